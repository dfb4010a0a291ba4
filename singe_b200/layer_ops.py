"""What the mixers of a layer-list decoder share: the library's entry points behind one activation type, and one step's rows
as the mixers read them."""
from __future__ import annotations

from dataclasses import dataclass, field

from . import kernel_sys as ks

FEW_TOKENS = 8                   # a sequence with at most this many new tokens takes the decode kernels


def round_up(value: int, multiple: int) -> int:
    return (value + multiple - 1) // multiple * multiple


class Ops:
    """The library's entry points for one activation type, and buffers laid out the way they want them (rows of whole
    16-byte pieces)."""

    def __init__(self, dtype: str):
        import torch

        if dtype not in ("bfloat16", "float32"):
            raise ValueError(f"activation type {dtype}")
        self.torch = torch
        self.dtype = getattr(torch, dtype)
        self.is_bf16 = dtype == "bfloat16"
        self.suffix = "bf16" if self.is_bf16 else "f32"

    def call(self, name: str, *arguments) -> None:
        code = getattr(ks.lib(), name)(*[a.data_ptr() if hasattr(a, "data_ptr") else a for a in arguments])
        if code != ks.OK:
            raise RuntimeError(f"{name}: status {code} ({ks.status_string(code)})")

    def rows(self, rows: int, columns: int):
        """[rows, columns] of the activation type with padded row stride."""
        return self.torch.empty((rows, round_up(columns, 8)), dtype=self.dtype, device="cuda")[:, :columns]

    def weight(self, array):
        """A matrix on the device with padded row stride, or a vector; the padding is zero."""
        torch = self.torch
        tensor = torch.as_tensor(array).to("cuda").to(self.dtype)
        if tensor.dim() < 2:
            return tensor.contiguous()
        out = torch.zeros((tensor.shape[0], round_up(tensor.shape[1], 8)), dtype=self.dtype, device="cuda")
        out[:, : tensor.shape[1]] = tensor
        return out[:, : tensor.shape[1]]

    def linear(self, stream, out, x, weight, activation: int = 0) -> None:
        m, k = x.shape
        n = weight.shape[0]
        if self.is_bf16:
            self.call("singe_linear_bf16", stream, out, x, weight, m, n, k, x.stride(0), weight.stride(0), out.stride(0),
                      activation, ks.HINT_STABLE_WEIGHTS)
        else:
            self.call("singe_linear_f32", stream, out, x, weight, m, n, k, x.stride(0), weight.stride(0), out.stride(0),
                      activation)

    def linear_f32_out(self, stream, out, x, weight) -> None:
        """f32 results whatever the activation type (logits)."""
        m, k = x.shape
        n = weight.shape[0]
        if self.is_bf16:
            self.call("singe_matmul_bf16_f32", stream, out, x, weight, m, n, k, x.stride(0), weight.stride(0),
                      out.stride(0), 0, 1)
        else:
            self.linear(stream, out, x, weight)

    def scalars(self, array):
        """Constants that enter f32 arithmetic whatever the activation type."""
        return self.torch.as_tensor(array).to("cuda").float().contiguous()

    def gate_up_weight(self, gate, up):
        """The weights of a gated feed-forward the way ``gated_linear_unit`` wants them: rows of the two in turn for the
        GEMM that applies the activation in its epilogue, one after the other otherwise."""
        torch = self.torch
        gate, up = torch.as_tensor(gate), torch.as_tensor(up)
        return self.weight(torch.stack([gate, up], 1).flatten(0, 1) if self.is_bf16 else torch.cat([gate, up]))

    def gated_linear_unit(self, stream, out, x, gate_up) -> None:
        """out = silu(gate x) * (up x)"""
        if self.is_bf16:
            self.linear(stream, out, x, gate_up, activation=1)
            return
        width = gate_up.shape[0] // 2
        both = self.rows(x.shape[0], 2 * width)
        self.linear(stream, both, x, gate_up)
        self.call("singe_silu_mul_f32", stream, out, out.stride(0), both, both.data_ptr() + width * both.element_size(),
                  both.stride(0), x.shape[0], width)

    def head_linear(self, stream, out, x, weight, heads: int, gate=None) -> None:
        """out[t, h] = x[t, h] . weight[h]^T (* sigmoid(gate[t, h])); x and out hold the heads side by side, weight stacks
        them [heads, columns, reduction]."""
        columns, reduction = weight.shape[1], weight.shape[2]
        arguments = [stream, out, x, weight, x.shape[0], heads, columns, reduction, x.stride(0), x.shape[1] // heads,
                     weight.stride(1), weight.stride(0) // weight.stride(1), out.stride(0), out.shape[1] // heads,
                     gate, 0 if gate is None else gate.stride(0)]
        if self.is_bf16:
            arguments.append(ks.HINT_STABLE_WEIGHTS)
        self.call(f"singe_head_linear_{self.suffix}", *arguments)

    def add_layer_norm(self, stream, residual, delta, normed, weight, eps: float) -> None:
        self.call(f"singe_add_layer_norm_{self.suffix}", stream, residual, delta,
                  0 if delta is None else delta.stride(0), normed, 0 if normed is None else normed.stride(0), weight,
                  residual.shape[0], residual.shape[1], eps)


# ------------------------------------------------------------------------------------------------
# one step's rows, as the mixers read them
# ------------------------------------------------------------------------------------------------

@dataclass
class StepRows:
    """Device inputs of a step.  int64: tokens, positions, pages, slots per packed row and the paging lists of the
    Tensor-surface attention; int32: each sequence's first row, new tokens and earlier tokens, the block table, and the
    rows that take the decode attention with the sequence and the number of visible keys of each."""
    count: int
    tokens: object
    pages: object
    slots: object
    query_offsets: object
    page_offsets: object
    page_list: object
    last_page_lengths: object
    first: object
    fresh_tokens: object
    context: object
    table: object
    positions: object
    sequence_of: object       # int32: the sequence of each row
    row_lens: object          # int32: keys up to and including each row's token, 0 for an idle row
    longest: int              # most new tokens of a sequence
    short_rows: object        # int32 [n], or None: row i of the step is query i
    short_sequences: object
    short_lens: object
    short_count: int
    expanded: dict = field(default_factory=dict)   # window -> ExpandedRows of the longer sequences
    blocks: dict = field(default_factory=dict)     # heads -> BlockRows of the longer sequences
    chunks: dict = field(default_factory=dict)     # chunk size -> ChunkRows of the longer sequences
    whole: object = None                           # BlockRows of the longer sequences, one segment each


@dataclass
class ExpandedRows:
    """What the prompt attention reads for one window: the cache rows whose keys and values it needs, packed sequence by
    sequence, and each sequence's lengths and offsets."""
    gather: object
    keys: int
    lens_q: object
    lens_kv: object
    offsets_q: object
    offsets_kv: object
    sequences: int


@dataclass
class BlockRows:
    """What the recurrence's prompt kernel reads: the blocks of the longer sequences and the segments that run side by side."""
    rows: object
    tokens: object
    blocks: int
    segments: object
    last: object
    count: int
    cut: bool


@dataclass
class ChunkRows:
    """What the prompt attention reads when every token sees its own chunk only: each (sequence, chunk) piece of the step is a
    sequence of its own, with keys packed piece by piece.  ``packed`` is each token's packed row (negative: its sequence takes
    the decode attention), ``cached`` whether a later step or this step's decode attention reads the token from the cache, and
    ``moved`` -> ``moved_to`` the cache rows of earlier tokens that pieces begin with."""
    packed: object
    cached: object
    keys: int
    moved: object
    moved_to: object
    lens_q: object
    lens_kv: object
    offsets_q: object
    offsets_kv: object
    pieces: int


def plan_chunks(size: int, context, fresh, first, long):
    """The pieces of a step's longer sequences: host arrays of ``ChunkRows`` by field, and the (sequence, position) pairs of the
    cached tokens to move.  ``context``, ``fresh`` and ``first`` are per sequence; ``long`` lists the longer ones."""
    import numpy as np

    rows = int(np.maximum(fresh, 1).sum())
    packed, cached = np.full(rows, -1, dtype=np.int64), np.ones(rows, dtype=np.uint8)
    pieces, moved, moved_to, keys = [], [], [], 0
    for b in long:
        start, end = int(context[b]), int(context[b] + fresh[b])
        last_chunk = end // size * size   # what a later token may still see
        at = start
        while at < end:
            begin = at // size * size
            stop = min(begin + size, end)
            row = int(first[b]) + at - start
            for position in range(begin, at):
                moved.append((b, position))
                moved_to.append(keys + position - begin)
            packed[row: row + stop - at] = keys + np.arange(at - begin, stop - begin)
            if stop <= last_chunk:
                cached[row: row + stop - at] = 0
            pieces.append((stop - at, stop - begin, row, keys))
            keys += stop - begin
            at = stop
    pieces = np.asarray(pieces, dtype=np.int64).reshape(-1, 4)
    return {"packed": packed, "cached": cached, "keys": keys, "moved": moved, "moved_to": np.asarray(moved_to, dtype=np.int64),
            "lens_q": pieces[:, 0], "lens_kv": pieces[:, 1], "offsets_q": pieces[:, 2], "offsets_kv": pieces[:, 3]}
