"""What every decoder here shares: the page table, the step's device inputs, graph capture, and the adapter the
generation loop drives.

  ``PageTable`` / ``DecodeStep``   singe/src/nn/decode/step.rs:131-475
  ``PagedDecoder``                 a model whose step is planned by a page table: status checks, the persistent inputs of
                                   a one-token-per-sequence step, its CUDA graph
  ``CachedDecoder``                the reference's ``Decoder`` trait over such a model (singe/src/generation/mod.rs:25-52)
"""
from __future__ import annotations

from dataclasses import dataclass

import numpy as np

from . import kernel_sys as ks


# ------------------------------------------------------------------------------------------------
# PageTable: singe/src/nn/decode/step.rs:131-475 (pure host integer planning)
# ------------------------------------------------------------------------------------------------

class PageTableError(ValueError):
    pass


@dataclass
class DecodeStep:
    """The paging tensors of one step (singe/src/nn/decode/step.rs:13-30), as int64 numpy arrays."""
    tokens: np.ndarray
    positions: np.ndarray
    write_pages: np.ndarray
    write_slots: np.ndarray
    query_offsets: np.ndarray
    page_offsets: np.ndarray
    pages: np.ndarray
    last_page_lengths: np.ndarray
    last_rows: np.ndarray
    real_tokens: np.ndarray
    sequence_ids: np.ndarray

    def wanted_rows(self, want) -> np.ndarray:
        """Rows of the step that hold the tokens at the places ``want[sequence]`` of each sequence's new tokens."""
        rows = []
        for sequence, places in enumerate(want):
            for place in places:
                if not 0 <= place < self.real_tokens[sequence]:
                    raise PageTableError("wanted token")
                rows.append(int(self.query_offsets[sequence]) + int(place))
        return np.asarray(rows, dtype=np.int64)


class PageTable:
    """Hands out cache pages to sequences in increasing order from page zero and writes each step's paging
    tensors.  After the pages sequences can hold comes one scratch page that held/idle rows and padding write.

    ``window`` (0: none) is the most tokens any layer looks back over, the token itself included: a page that no later
    token of its sequence can see goes back to the pool at the sequence's next step, and the scratch page takes its
    place in the sequence's list.  ``chunks`` are the sizes of the chunks of positions that layers see instead of a window: such
    a layer sees nothing before the chunk the token stands in."""

    def __init__(self, sequences: int, capacity: int, page_size: int, pool: int, window: int = 0, chunks=()):
        self.page_size = page_size
        self.capacity = capacity
        self.pool = pool
        self.window = window
        self.chunks = tuple(chunks)
        self.padding = 0
        self.free: list[int] = []
        self.pages: list[list[int]] = [[] for _ in range(sequences)]
        self.lengths: list[int] = [0] * sequences
        self.reset()

    @classmethod
    def create(cls, sequences: int, capacity: int, page_size: int) -> "PageTable":
        if sequences == 0 or capacity <= 0 or page_size <= 0:
            raise PageTableError("page table size")
        return cls(sequences, capacity, page_size, sequences * ((capacity - 1) // page_size + 1))

    @classmethod
    def create_shared(cls, sequences: int, capacity: int, page_size: int, cache_tokens: int,
                      window: int = 0, chunks=()) -> "PageTable":
        if sequences == 0 or capacity <= 0 or page_size <= 0 or cache_tokens <= 0 or window < 0 or any(c <= 0 for c in chunks):
            raise PageTableError("page table size")
        return cls(sequences, capacity, page_size, (cache_tokens - 1) // page_size + 1, window, chunks)

    def with_padding(self, padding: int) -> "PageTable":
        self.padding = padding
        return self

    def reset(self) -> None:
        self.free = list(range(self.pool - 1, -1, -1))
        self.pages = [[] for _ in self.pages]
        self.lengths = [0] * len(self.lengths)

    def release(self, sequence: int) -> None:
        if not 0 <= sequence < len(self.pages):
            raise PageTableError("decoder sequence")
        self.free.extend(page for page in reversed(self.pages[sequence]) if page != self.pool)
        self.pages[sequence] = []
        self.lengths[sequence] = 0

    def free_pages(self) -> int:
        return len(self.free)

    def page_count(self) -> int:
        return self.pool + 1

    @property
    def scratch_page(self) -> int:
        return self.pool

    def _unseen(self, row: int) -> list:
        """Places in a sequence's page list that its next token and all after it cannot see any more."""
        if self.window == 0 and not self.chunks:
            return []
        length = self.lengths[row]   # the next token's position
        oldest = [length // size * size for size in self.chunks]
        if self.window > 0:
            oldest.append(max(length - self.window + 1, 0))
        dead = min(oldest) // self.page_size
        return [place for place in range(dead) if self.pages[row][place] != self.pool]

    def table_length(self) -> int:
        held = self.pool
        if self.window > 0 or self.chunks:  # lists also name the scratch page, once for every page given back
            held = max(held, len(self.pages) * ((self.capacity - 1) // self.page_size + 1))
        return held + len(self.pages) + (self.padding + self.page_size - 1) // self.page_size

    @staticmethod
    def step_tokens(tokens) -> int:
        return sum(max(len(t), 1) for t in tokens)

    def step(self, tokens) -> DecodeStep:
        return self.step_padded(tokens, self.step_tokens(tokens))

    def step_padded(self, tokens, total: int) -> DecodeStep:
        sequences = len(self.pages)
        if len(tokens) != sequences or all(len(t) == 0 for t in tokens):
            raise PageTableError("decode step needs a slice for every sequence, and tokens in one")
        padding = total - self.step_tokens(tokens)
        if padding < 0:
            raise PageTableError("a decode step is padded to fewer rows than it has")
        if padding > self.padding:
            raise PageTableError("a decode step is padded past what its page table allows")
        padded = max(i for i, t in enumerate(tokens) if len(t) > 0)
        for length, t in zip(self.lengths, tokens):
            if length + len(t) > self.capacity:
                raise PageTableError("decoder cache capacity")
        fresh = 0
        for length, held, t in zip(self.lengths, self.pages, tokens):
            if len(t) > 0:
                end = length + len(t)
                fresh += max((end - 1) // self.page_size + 1 - len(held), 0)
        unseen = {row: self._unseen(row) for row, t in enumerate(tokens) if len(t) > 0}
        if fresh > len(self.free) + sum(len(places) for places in unseen.values()):
            raise PageTableError("decoder cache pages")
        for row, places in unseen.items():
            self.free.extend(self.pages[row][place] for place in reversed(places))
            for place in places:
                self.pages[row][place] = self.pool

        flat, positions, write_pages, write_slots = [], [], [], []
        query_offsets, last_rows, real_tokens, sequence_ids, visible = [0], [], [], [], []
        for row, t in enumerate(tokens):
            held = self.pages[row]
            for token in t:
                position = self.lengths[row]
                page = position // self.page_size
                if page == len(held):
                    held.append(self.free.pop())
                flat.append(int(token))
                positions.append(position)
                write_pages.append(held[page])
                write_slots.append(position % self.page_size)
                self.lengths[row] += 1
            if len(t) == 0:
                flat.append(0)
                positions.append(min(self.lengths[row], self.capacity - 1))
                write_pages.append(self.pool)
                write_slots.append(0)
            last = len(flat) - 1
            keys = self.lengths[row]
            if row == padded:
                for position in range(self.lengths[row], self.lengths[row] + padding):
                    flat.append(0)
                    positions.append(min(position, self.capacity - 1))
                    write_pages.append(self.pool)
                    write_slots.append(position % self.page_size)
                keys += padding
            visible.append(keys)
            sequence_ids.extend([row] * (len(flat) - len(sequence_ids)))
            query_offsets.append(len(flat))
            last_rows.append(last)
            real_tokens.append(len(t))

        pages, page_offsets, last_page_lengths = [], [0], []
        for held, seen in zip(self.pages, visible):
            if seen == 0:
                pages.append(self.pool)
                last_page_lengths.append(1)
            else:
                used = (seen - 1) // self.page_size + 1
                kept = min(used, len(held))
                pages.extend(held[:kept])
                pages.extend([self.pool] * (used - kept))
                last_page_lengths.append((seen - 1) % self.page_size + 1)
            page_offsets.append(len(pages))
        pages.extend([0] * (self.table_length() - len(pages)))
        as_array = lambda values: np.asarray(values, dtype=np.int64)
        return DecodeStep(as_array(flat), as_array(positions), as_array(write_pages), as_array(write_slots),
                          as_array(query_offsets), as_array(page_offsets), as_array(pages),
                          as_array(last_page_lengths), as_array(last_rows), as_array(real_tokens),
                          as_array(sequence_ids))

    def place_prompts(self, lengths) -> None:
        """Advances every sequence by ``lengths[b]`` tokens without building step tensors (bulk prompt placement)."""
        for row, count in enumerate(lengths):
            if self.lengths[row] + count > self.capacity:
                raise PageTableError("decoder cache capacity")
            need = (self.lengths[row] + count - 1) // self.page_size + 1 - len(self.pages[row]) if count > 0 else 0
            if need > len(self.free):
                raise PageTableError("decoder cache pages")
            for _ in range(max(need, 0)):
                self.pages[row].append(self.free.pop())
            self.lengths[row] += count


# ------------------------------------------------------------------------------------------------
# decoders
# ------------------------------------------------------------------------------------------------

class PagedDecoder:
    """Base of the decoders.  A subclass builds its weights and caches, calls ``_init_step_inputs``, and provides
    ``forward()`` (one token per sequence, reading the persistent inputs) and ``step_tokens()`` (steps of any shape)."""

    def _init_step_inputs(self, table: PageTable, sequences: int, capacity: int, page_size: int) -> None:
        """The page table and the persistent device inputs of a one-token-per-sequence step."""
        import torch

        self.torch = torch
        self.table = table
        self.sequences = sequences
        self.capacity = capacity
        self.stride = (capacity + page_size - 1) // page_size
        i64, i32 = torch.int64, torch.int32
        zeros = lambda shape, dtype: torch.zeros(shape, dtype=dtype, device="cuda")
        self.d_tokens = zeros(sequences, i64)
        self.d_positions = zeros(sequences, i64)
        self.d_pages = zeros(sequences, i64)
        self.d_slots = zeros(sequences, i64)
        self.d_lens = zeros(sequences, i32)
        self.d_table = zeros((sequences, self.stride), i32)
        self.h_table = np.zeros((sequences, self.stride), dtype=np.uint32)
        self.status = zeros(1, i32)
        self.best_value = torch.empty(sequences, dtype=torch.float32, device="cuda")
        self.best_index = torch.empty(sequences, dtype=i64, device="cuda")
        self.next_tokens = torch.empty(sequences, dtype=i64, device="cuda")
        self.graph = None

    def _check(self, code: int, where: str) -> None:
        if code != ks.OK:
            raise RuntimeError(f"{where}: status {code} ({ks.status_string(code)})")

    def _stream(self) -> int:
        return int(self.torch.cuda.current_stream().cuda_stream)

    def _refresh_block_table(self) -> None:
        for b, held in enumerate(self.table.pages):
            self.h_table[b, : len(held)] = held
        self.d_table.copy_(self.torch.from_numpy(self.h_table.view(np.int32)))

    def plan(self, tokens) -> DecodeStep:
        """One token per sequence -> the step's paging tensors, uploaded into the persistent device buffers."""
        return self._plan_lists([[int(t)] for t in tokens])

    def _plan_lists(self, tokens) -> DecodeStep:
        """The same for at most one token per sequence; an idle row sees no key."""
        torch = self.torch
        step = self.table.step(tokens)
        self._refresh_block_table()
        self.d_tokens.copy_(torch.from_numpy(step.tokens))
        self.d_positions.copy_(torch.from_numpy(step.positions))
        self.d_pages.copy_(torch.from_numpy(step.write_pages))
        self.d_slots.copy_(torch.from_numpy(step.write_slots))
        self.d_lens.copy_(torch.from_numpy(np.where(step.real_tokens > 0, step.positions + 1, 0).astype(np.int32)))
        return step

    def forward(self) -> None:
        raise NotImplementedError

    def step_tokens(self, tokens, want=None):
        raise NotImplementedError

    def capture(self) -> None:
        """Captures ``forward`` into a CUDA graph that later steps replay (the reference replays a captured
        step the same way, singe/src/generation/mod.rs:529-579)."""
        torch = self.torch
        side = torch.cuda.Stream()
        side.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(side):
            self.forward()  # warm-up outside capture: loads modules, sizes nothing (all buffers are preallocated)
        torch.cuda.current_stream().wait_stream(side)
        torch.cuda.synchronize()
        self.graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(self.graph):
            self.forward()

    def run(self) -> None:
        """The planned one-token step: the captured graph if there is one."""
        if self.graph is not None:
            self.graph.replay()
        else:
            self.forward()

    def step(self, tokens) -> "object":
        """Plans and runs one decode step; returns the device tensor of greedy next tokens [sequences]."""
        self.plan(tokens)
        self.run()
        return self.next_tokens

    def reset(self) -> None:
        self.table.reset()

    def release(self, sequence: int) -> None:
        self.table.release(sequence)


class CachedDecoder:
    """A ``PagedDecoder`` behind the reference's ``Decoder`` trait (singe/src/generation/mod.rs:25-52), which is what
    ``singe_b200.generation`` drives: ``sequences()``, ``step(tokens)``, ``reset()``, ``release(row)``,
    ``largest_chunk()``.  Prompt steps read at most the largest prompt chunk of extra tokens (16, 64, 256, ... 1024,
    ``PromptChunks``, :367-417)."""

    def __init__(self, model: PagedDecoder, prompt_chunks=None):
        from .generation import PromptChunks

        self.model = model
        self.chunks = (prompt_chunks or PromptChunks.STANDARD).sizes(model.capacity)

    def sequences(self) -> int:
        return self.model.sequences

    def step(self, tokens):
        return self.model.step_tokens(tokens)

    def reset(self) -> None:
        self.model.reset()

    def release(self, sequence: int) -> None:
        self.model.release(sequence)

    def largest_chunk(self):
        return self.chunks[-1] if self.chunks else 0
