"""Decoder whose configuration lists its layers one by one, each with its own mixer and an optional feed-forward.

``HybridDecoder`` is a ``PagedDecoder``: the page table, the one-token step and its CUDA graph, the generation loop and
the checkpoint reader are the ones every decoder here uses.  Its parts:

  ``LatentAttention``   attention over a low-rank latent of the context.  The cache holds one normalised latent row per
                        token, shared by all heads, behind the page table; a sliding window bounds what a token sees and
                        lets the page table take unseen pages back.
  ``GatedLinear``       gated linear attention: a recurrent state per sequence, [heads, dim, vdim] in f32, in the
                        sequence's row; a sequence's first token starts it from zero, so a row that is used again needs
                        no clearing.
  ``ParallelMixer``     chunked attention and the gated delta rule side by side (``parallel_mixer``)
  feed-forward          down(relu(up(h))^2) or down(silu(gate(h)) * up(h))
  residual              one stream with layer norms, or several with RMS norms (``residual``)

A layer may borrow another layer's weights; its cache or state is always its own.  The residual streams and all norms
are f32.  ``dtype`` "bfloat16" keeps weights and activations in bf16 (f32 accumulation, tensor-core kernels); "float32"
computes everything in true 32-bit with the library's f32 kernels.

Latent attention has two forms of the same product.  Per head, score = (W_uq c_q) . (W_uk c) and value = W_uv c:
  absorbed   q' = W_uk^T q, then attention of q' over the latents themselves, then W_uv on the attended latent: reads only
             the cache, for steps of few tokens per sequence;
  expanded   k and v of every visible latent are computed by one GEMM and attended on the tensor core: for prompts.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import numpy as np

from . import kernel_sys as ks
from .decoder import PagedDecoder, PageTable
from .layer_ops import FEW_TOKENS, BlockRows, ChunkRows, ExpandedRows, Ops, StepRows, plan_chunks, round_up
from .parallel_mixer import ParallelConfig, ParallelMixer
from .residual import LayerNormResidual, StreamResidual, Sublayer

EXPANDED_HEAD_SIZES = (64, 128)  # head sizes of the tensor-core prompt attention; smaller heads are padded with zeros
ABSORBED_LATENT_LIMIT = 512      # widest latent the tensor-core decode attention takes
BLOCK_TOKENS = 16                # tokens of a block of the recurrence's prompt kernel
LEAST_SEGMENT = 8                # blocks a long sequence's segments have at least


# ------------------------------------------------------------------------------------------------
# configuration
# ------------------------------------------------------------------------------------------------

@dataclass(frozen=True)
class LatentAttentionConfig:
    heads: int
    dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    window: int


@dataclass(frozen=True)
class GatedLinearConfig:
    heads: int
    dim: int
    vdim: int
    rank: int      # of the decay projection
    tau: float


@dataclass(frozen=True)
class LayerConfig:
    mixer: object
    ffn: int = 0               # 0: the layer has no feed-forward
    weights_of: int | None = None
    gated: bool = False        # the feed-forward is silu(gate) * up instead of relu(up)^2


@dataclass
class HybridConfig:
    layers: list = field(default_factory=list)
    width: int = 0
    vocab: int = 0
    eps: float = 1e-6
    page_size: int = 64        # a page of this size is one tile of the decode attention over latents
    streams: int = 0           # 0: one residual stream with layer norms; else that many, with RMS norms
    logit_scale: float = 1.0   # with streams

    def owner(self, index: int) -> int:
        """The layer whose weights layer ``index`` uses."""
        seen = {index}
        while self.layers[index].weights_of is not None:
            index = self.layers[index].weights_of
            if not 0 <= index < len(self.layers) or index in seen:
                raise ValueError(f"layer {index}: borrowed weights lead nowhere")
            seen.add(index)
        return index

    def window(self) -> int:
        """The most tokens any layer with a sliding window looks back over through the cache; 0 when chunks alone bound it."""
        return max((layer.mixer.window for layer in self.layers if isinstance(layer.mixer, LatentAttentionConfig)),
                   default=0 if self.chunks() else 1)

    def chunks(self) -> list:
        """The chunk sizes of the layers whose tokens see their own chunk."""
        return sorted({layer.mixer.left.chunk for layer in self.layers if isinstance(layer.mixer, ParallelConfig)})


def plan_segments(blocks_of, heads: int, sms: int):
    """Cuts each sequence's blocks into segments.  A cut costs a second pass over all but a sequence's last segment, so
    only steps whose (sequence, head) pairs leave SMs idle are cut, into about three (segment, head) pairs per SM.  Returns rows of
    (place in ``blocks_of``, first block, blocks, earlier segments of the sequence, last of the sequence)."""
    total = sum(blocks_of)
    size = total
    if len(blocks_of) * heads < sms:
        size = max(LEAST_SEGMENT, -(-total // max(3 * sms // heads, 1)))
    rows, first = [], 0
    for place, blocks in enumerate(blocks_of):
        pieces = -(-blocks // size)
        each = -(-blocks // pieces)
        done = 0
        while done < blocks:
            taken = min(each, blocks - done)
            rows.append((place, first + done, taken, done // each, int(done + taken == blocks)))
            done += taken
        first += blocks
    return rows


# ------------------------------------------------------------------------------------------------
# mixers
# ------------------------------------------------------------------------------------------------

class LatentAttention:
    """Weights of one latent-attention layer and its step.  ``source`` maps tensor names to arrays."""

    def __init__(self, config: LatentAttentionConfig, source, ops: Ops, eps: float):
        torch = ops.torch
        self.config, self.ops, self.eps = config, ops, eps
        c = config
        take = lambda name: torch.as_tensor(source(name)).to("cuda").to(ops.dtype)
        widest = max(c.dim, c.vdim)
        # the tensor-core kernels: heads of a size the prompt attention has, latents the decode attention takes
        self.tiled = ops.is_bf16 and widest <= EXPANDED_HEAD_SIZES[-1] and c.kv_rank <= ABSORBED_LATENT_LIMIT
        if self.tiled:
            self.key_size = self.value_size = next(size for size in EXPANDED_HEAD_SIZES if widest <= size)
            self.latent = round_up(c.kv_rank, 64)
        else:
            unit = 8 if ops.is_bf16 else 1   # 16-byte rows for the bf16 GEMM
            self.key_size, self.value_size = round_up(c.dim, unit), round_up(c.vdim, unit)
            self.latent = round_up(c.kv_rank, unit)
        self.down = ops.weight(torch.cat([take("dq"), take("dkv"), take("g")]))
        self.q_norm, self.kv_norm = ops.weight(take("dq.norm")), ops.weight(take("dkv.norm"))
        # every head's rows (or columns) padded to the head size, the latent's columns to the cache row
        padded = lambda array, size: torch.nn.functional.pad(
            array.reshape(c.heads, -1, array.shape[1]), (0, 0, 0, size - array.shape[0] // c.heads))
        self.uq = ops.weight(padded(take("uq"), self.key_size).reshape(c.heads * self.key_size, c.q_rank))
        pad_latent = lambda array: torch.nn.functional.pad(array, (0, self.latent - c.kv_rank))
        uk, uv = pad_latent(padded(take("uk"), self.key_size)), pad_latent(padded(take("uv"), self.value_size))
        self.absorb = uk.transpose(1, 2).contiguous()          # [heads, latent, key_size]
        if self.tiled:                                         # [2 * heads * size, latent]: keys, then values
            self.expand = torch.cat([uk, uv]).reshape(2 * c.heads * self.key_size, self.latent).contiguous()
            self.uv = self.expand[c.heads * self.key_size:].view(c.heads, self.value_size, self.latent)
        else:
            self.expand, self.uv = None, uv.contiguous()
        out = take("o")
        out = torch.nn.functional.pad(out.reshape(out.shape[0], c.heads, c.vdim), (0, self.value_size - c.vdim))
        self.out = ops.weight(out.reshape(out.shape[0], c.heads * self.value_size))

    def new_cache(self, table: PageTable, sequences: int):
        torch = self.ops.torch
        return torch.zeros((table.page_count(), table.page_size, 1, self.latent), dtype=self.ops.dtype, device="cuda")

    def scratch(self, rows: int, key_bound: int):
        """Partial results of the split decode attention for ``rows`` queries over at most ``key_bound`` keys."""
        if not self.tiled:
            return None
        torch, c = self.ops.torch, self.config
        splits = int(ks.lib().singe_latent_decode_splits(rows, c.heads, self.latent, min(key_bound, c.window)))
        attn = torch.empty((rows, splits, c.heads, self.latent), dtype=torch.float32, device="cuda")
        lse = torch.empty((rows, splits, c.heads), dtype=torch.float32, device="cuda")
        return splits, attn, lse

    def run(self, stream, step: StepRows, normed, cache, delta, status, scratch=None) -> None:
        """delta = W_o of the gated heads' outputs for the rows of ``normed``."""
        ops, c = self.ops, self.config
        t = normed.shape[0]
        pages, page_size = cache.shape[0], cache.shape[1]
        projected = ops.rows(t, c.q_rank + c.kv_rank + c.heads)
        ops.linear(stream, projected, normed, self.down)
        latent_query = ops.rows(t, c.q_rank)
        ops.call(f"singe_latent_norm_cache_write_{ops.suffix}", stream, latent_query, latent_query.stride(0), cache,
                 self.latent, projected, projected.stride(0), self.q_norm, c.q_rank, self.kv_norm, c.kv_rank, step.pages,
                 step.slots, t, pages, page_size, self.eps, status)
        query = ops.rows(t, c.heads * self.key_size)
        ops.linear(stream, query, latent_query, self.uq)
        gate = projected[:, c.q_rank + c.kv_rank:]
        attended = ops.rows(t, c.heads * self.value_size)
        if not self.tiled:
            self._general(stream, step, query, cache, gate, attended, status)
        else:
            if c.window in step.expanded:
                self._expanded(stream, step.expanded[c.window], query, cache, gate, attended, status)
            if step.short_count > 0:
                self._absorbed(stream, step, query, cache, gate, attended, status, scratch)
        ops.linear(stream, delta, attended, self.out)

    def _general(self, stream, step, query, cache, gate, attended, status) -> None:
        """Absorbed attention of every row on the general kernel: any sizes, either activation type."""
        ops, c = self.ops, self.config
        t = query.shape[0]
        # rows without padding, as the attention wants them
        latent_queries, latents = ops.torch.empty((2, t, c.heads * self.latent), dtype=ops.dtype, device="cuda")
        ops.head_linear(stream, latent_queries, query, self.absorb, c.heads)
        lse = ops.torch.empty((t, c.heads), dtype=ops.torch.float32, device="cuda")
        ops.call(f"singe_paged_attention_{ops.suffix}", stream, latents, lse, latent_queries, cache, cache,
                 step.query_offsets, step.page_offsets, step.page_list, step.last_page_lengths, 8, t, c.heads, 1,
                 self.latent, cache.shape[1], cache.shape[0], step.last_page_lengths.numel(), step.page_list.numel(),
                 c.scale, 1, c.window, status)
        ops.head_linear(stream, attended, latents, self.uv, c.heads, gate)

    def _absorbed(self, stream, step, query, cache, gate, attended, status, scratch) -> None:
        """Absorbed attention of the rows whose sequences have few new tokens."""
        ops, c = self.ops, self.config
        rows, n = step.short_rows, step.short_count
        values = attended
        if rows is not None:
            query, gate = query.index_select(0, rows), gate.index_select(0, rows)
            values = ops.rows(n, c.heads * self.value_size)
        latent_queries, latents = ops.rows(n, c.heads * self.latent), ops.rows(n, c.heads * self.latent)
        ops.head_linear(stream, latent_queries, query, self.absorb, c.heads)
        splits, attn, lse = scratch or self.scratch(n, step.table.shape[1] * cache.shape[1])
        ops.call("singe_latent_decode_bf16", stream, latents, attn, lse, latent_queries, cache, step.short_sequences,
                 step.short_lens, step.table, n, c.heads, self.latent, cache.shape[1], cache.shape[0],
                 step.table.shape[0], step.table.shape[1], c.window, splits, c.scale, status)
        ops.head_linear(stream, values, latents, self.uv, c.heads, gate)
        if rows is not None:
            attended.index_copy_(0, rows, values)

    def _expanded(self, stream, rows: ExpandedRows, query, cache, gate, attended, status) -> None:
        ops, c, size = self.ops, self.config, self.key_size
        torch = ops.torch
        latents = torch.empty((rows.keys, self.latent), dtype=ops.dtype, device="cuda")
        ops.call("singe_gather_rows", stream, latents, cache, rows.gather, rows.keys, self.latent * 2,
                 cache.shape[0] * cache.shape[1], status)
        keys_values = torch.empty((rows.keys, 2 * c.heads * size), dtype=ops.dtype, device="cuda")
        ops.linear(stream, keys_values, latents, self.expand)
        lse = torch.empty((query.shape[0], c.heads), dtype=torch.float32, device="cuda")
        ops.call("singe_windowed_prefill_attention_bf16", stream, attended, lse, query, keys_values,
                 keys_values.data_ptr() + c.heads * size * 2, keys_values.stride(0), rows.lens_q, rows.lens_kv,
                 rows.offsets_q, rows.offsets_kv, gate, gate.stride(0), rows.sequences, query.shape[0], rows.keys,
                 c.heads, c.heads, size, c.window, c.scale)


class GatedLinear:
    """Weights of one gated-linear-attention layer and its step."""

    def __init__(self, config: GatedLinearConfig, source, ops: Ops, eps: float):
        torch = ops.torch
        self.config, self.ops, self.eps = config, ops, eps
        take = lambda name: torch.as_tensor(source(name)).to("cuda").to(ops.dtype)
        self.project = ops.weight(torch.cat([take("q"), take("k"), take("v"), take("g"), take("a1")]))
        self.decay, self.bias, self.norm = take("a2").contiguous(), take("a2.b").contiguous(), take("norm").contiguous()
        self.out = ops.weight(take("o"))
        # the prompt kernel, for sizes it takes
        self.blocked = ops.is_bf16 and ks.lib().singe_gated_linear_prompt_scratch(config.heads, config.dim, config.vdim, 1, 1) > 0

    def new_cache(self, table: PageTable, sequences: int):
        c = self.config
        return self.ops.torch.zeros((sequences, c.heads, c.dim, c.vdim), dtype=self.ops.torch.float32, device="cuda")

    def scratch(self, rows: int, key_bound: int):
        return None

    def run(self, stream, step: StepRows, normed, state, delta, status, scratch=None) -> None:
        ops, c = self.ops, self.config
        t = normed.shape[0]
        projected = ops.rows(t, self.project.shape[0])
        ops.linear(stream, projected, normed, self.project)
        attended = ops.rows(t, c.heads * c.vdim)
        operands = [attended, attended.stride(0), projected, projected.stride(0), self.decay, self.bias, self.norm, state]
        sizes = [c.heads, c.dim, c.vdim, c.rank, c.tau, c.dim ** -0.5, self.eps]
        rows = step.blocks.get(c.heads) if self.blocked else None
        if rows is not None:
            scratch = ops.torch.empty(int(ks.lib().singe_gated_linear_prompt_scratch(c.heads, c.dim, c.vdim, rows.blocks,
                                                                                     rows.count)),
                                      dtype=ops.torch.uint8, device="cuda")
            ops.call("singe_gated_linear_prompt_bf16", stream, *operands, step.context, t, *sizes, rows.rows, rows.tokens,
                     rows.blocks, rows.segments, rows.last, rows.count, int(rows.cut), scratch)
        if rows is None or step.short_count > 0:
            ops.call(f"singe_gated_linear_step_{ops.suffix}", stream, *operands, step.first, step.fresh_tokens,
                     step.context, t, state.shape[0], *sizes, 0x7fffffff if rows is None else FEW_TOKENS)
        ops.linear(stream, delta, attended, self.out)


MIXERS = {LatentAttentionConfig: LatentAttention, GatedLinearConfig: GatedLinear, ParallelConfig: ParallelMixer}


# ------------------------------------------------------------------------------------------------
# decoder
# ------------------------------------------------------------------------------------------------

@dataclass
class _Layer:
    mixer: object
    first: Sublayer
    second: Sublayer = None
    up: object = None      # with gated: gate and up together
    down: object = None
    gated: bool = False


class HybridDecoder(PagedDecoder):
    """The decoder: weights, caches and states, and its steps.  ``weights`` maps tensor names to arrays (what
    ``singe_b200.checkpoint.load_hybrid`` returns); ``cache_tokens`` sizes a cache pool shared by the sequences
    (default: room for every sequence's whole capacity)."""

    def __init__(self, config: HybridConfig, sequences: int, capacity: int, weights: dict, dtype: str = "bfloat16",
                 cache_tokens: int | None = None):
        import torch

        self.config = config
        self.dtype = dtype
        self.ops = ops = Ops(dtype)
        whole = sequences * round_up(capacity, config.page_size)
        table = PageTable.create_shared(sequences, capacity, config.page_size, cache_tokens or whole, config.window(),
                                        config.chunks())
        self._init_step_inputs(table, sequences, capacity, config.page_size)
        take = lambda name: torch.as_tensor(weights[name])
        self.residual = (StreamResidual if config.streams else LayerNormResidual)(config, take, ops)
        built = {}
        for index, layer in enumerate(config.layers):
            if layer.weights_of is not None:
                continue
            prefix = f"l{index}."
            mixer = MIXERS[type(layer.mixer)](layer.mixer, lambda name, p=prefix: take(p + "mix." + name), ops, config.eps)
            norms = getattr(mixer, "output_norms", None)
            built[index] = _Layer(mixer, self.residual.sublayer(take, prefix, 1, norms), gated=layer.gated)
            if layer.ffn:
                built[index].second = self.residual.sublayer(take, prefix, 2)
                built[index].up = (ops.gate_up_weight(take(prefix + "mlp.gate"), take(prefix + "mlp.up")) if layer.gated
                                   else ops.weight(take(prefix + "mlp.up")))
                built[index].down = ops.weight(take(prefix + "mlp.down"))
        self.layers = [built[config.owner(index)] for index in range(len(config.layers))]
        self.caches = [layer.mixer.new_cache(table, sequences) for layer in self.layers]
        self.head = ops.weight(take("head"))
        # persistent inputs of the one-token step beyond those every decoder has
        i32, i64 = torch.int32, torch.int64
        zeros = lambda shape, kind: torch.zeros(shape, dtype=kind, device="cuda")
        self.d_first = torch.arange(sequences, dtype=i32, device="cuda")
        self.d_fresh = zeros(sequences, i32)
        self.d_context = zeros(sequences, i32)
        self.d_query_offsets = torch.arange(sequences + 1, dtype=i64, device="cuda")
        self.d_page_offsets = zeros(sequences + 1, i64)
        self.d_page_list = zeros(table.table_length(), i64)
        self.d_last_lengths = zeros(sequences, i64)
        self.logits = torch.empty((sequences, config.vocab), dtype=torch.float32, device="cuda")
        self.scratches = {id(layer): layer.mixer.scratch(sequences, self.stride * config.page_size)
                          for layer in built.values()}
        self.decode_rows = StepRows(sequences, self.d_tokens, self.d_pages, self.d_slots, self.d_query_offsets,
                                    self.d_page_offsets, self.d_page_list, self.d_last_lengths, self.d_first,
                                    self.d_fresh, self.d_context, self.d_table, self.d_positions, self.d_first,
                                    self.d_lens, 1, None, self.d_first, self.d_lens, sequences)
        self.sms = torch.cuda.get_device_properties(0).multi_processor_count
        self.trail = None   # set to a list to collect the residual stream after every layer (for inspection)

    def fill_context(self, tokens_per_sequence: int, seed: int = 4) -> None:
        """Marks ``tokens_per_sequence`` tokens of every sequence as cached and fills caches and states with N(0,1) values
        (a benchmark's stand-in for a processed prompt)."""
        torch = self.torch
        self.table.place_prompts([tokens_per_sequence] * self.sequences)
        generator = torch.Generator(device="cuda").manual_seed(seed)
        for cache in self.caches:
            for part in cache if isinstance(cache, tuple) else (cache,):
                part.normal_(generator=generator)
        self._refresh_block_table()

    # ---- the layers, over a step of any shape ----

    def _layers(self, rows: StepRows, scratches):
        """Runs the layers; returns the final norm's output for the step's rows."""
        ops, c = self.ops, self.config
        stream = self._stream()
        t = rows.count
        normed = ops.rows(t, c.width)
        residual, done, delta = None, None, None   # done, delta: the sublayer whose output the residual has not taken in yet
        for layer, cache in zip(self.layers, self.caches):
            if done is None:
                residual = self.residual.start(stream, rows, layer.first, normed, self.status)
            else:
                self.residual.advance(stream, residual, delta, done, layer.first, normed)
            done = layer.first
            delta = ops.rows(t, c.width if done.output_norms is None else round_up(c.width, 8) + c.width)
            layer.mixer.run(stream, rows, normed, cache, delta, self.status, scratches.get(id(layer)))
            if layer.second is not None:
                self.residual.advance(stream, residual, delta, done, layer.second, normed)
                done, delta = layer.second, ops.rows(t, c.width)
                inner = ops.rows(t, layer.down.shape[1])
                if layer.gated:
                    ops.gated_linear_unit(stream, inner, normed, layer.up)
                else:
                    ops.linear(stream, inner, normed, layer.up, activation=2)
                ops.linear(stream, delta, inner, layer.down)
            if self.trail is not None:
                self.trail.append(self.residual.peek(stream, residual, delta, done))
        self.residual.finish(stream, residual, delta, done, normed)
        return normed

    def forward(self) -> None:
        """One token per sequence, from the persistent step inputs; idle rows have nothing in ``d_fresh``."""
        stream = self._stream()
        normed = self._layers(self.decode_rows, self.scratches)
        self.ops.linear_f32_out(stream, self.logits, normed, self.head)
        self.ops.call("singe_argmax_f32", stream, self.best_value, self.next_tokens, self.logits, self.logits.stride(0),
                      self.sequences, self.config.vocab, 0)

    def _plan_lists(self, tokens):
        step = super()._plan_lists(tokens)
        torch = self.torch
        to = lambda target, array: target.copy_(torch.from_numpy(np.ascontiguousarray(array)))
        to(self.d_fresh, step.real_tokens.astype(np.int32))
        to(self.d_context, (np.asarray(self.table.lengths) - step.real_tokens).astype(np.int32))
        to(self.d_page_offsets, step.page_offsets)
        to(self.d_page_list, step.pages)
        to(self.d_last_lengths, step.last_page_lengths)
        return step

    def capture(self) -> None:
        """The captured step must not leave anything behind: it is recorded with every row idle."""
        self.d_pages.fill_(self.table.scratch_page)
        for idle in (self.d_tokens, self.d_slots, self.d_lens, self.d_fresh):
            idle.zero_()
        super().capture()

    def step_tokens(self, tokens, want=None):
        """Extends each sequence with its ``tokens`` (an empty list leaves a row idle) and returns the logits of each
        sequence's last token, f32 [sequences, vocab]; with ``want`` (one list of places among its new tokens per
        sequence) the logits of those tokens, [wanted, vocab], in that order.  A step that cannot get its pages raises
        before anything changed."""
        torch = self.torch
        tokens = [[int(v) for v in t] for t in tokens]
        if all(len(t) <= 1 for t in tokens):
            step = self._plan_lists(tokens)
            self.run()
            return self.logits if want is None else self.logits[torch.from_numpy(step.wanted_rows(want)).cuda()]
        step = self.table.step(tokens)
        rows = self._upload(step)
        normed = self._layers(rows, {})
        picked = step.last_rows if want is None else step.wanted_rows(want)
        logits = torch.empty((len(picked), self.config.vocab), dtype=torch.float32, device="cuda")
        if len(picked) > 0:
            last = self.ops.rows(len(picked), self.config.width)
            last.copy_(normed.index_select(0, torch.from_numpy(picked).cuda()))
            self.ops.linear_f32_out(self._stream(), logits, last, self.head)
        return logits

    def _upload(self, step) -> StepRows:
        """The device inputs of a step of any shape: two copies, one per integer width."""
        torch, c = self.torch, self.config
        table = self.table
        lengths = np.asarray(table.lengths, dtype=np.int64)
        fresh = step.real_tokens
        context = lengths - fresh
        first = step.query_offsets[:-1]
        page_counts = np.asarray([max(len(held), 1) for held in table.pages])
        block_table = np.full((self.sequences, int(page_counts.max())), table.scratch_page, dtype=np.int64)
        for b, held in enumerate(table.pages):
            block_table[b, : len(held)] = held
        few = fresh <= FEW_TOKENS
        short = np.nonzero(few[step.sequence_ids])[0]
        sequences = step.sequence_ids[short]
        lens = np.where(fresh[sequences] > 0, step.positions[short] + 1, 0)
        narrow = {"first": first, "fresh": fresh, "context": context, "table": block_table.reshape(-1),
                  "short_sequences": sequences, "short_lens": lens}
        long = np.nonzero(~few)[0]
        windows = sorted({layer.mixer.window for layer in c.layers if isinstance(layer.mixer, LatentAttentionConfig)})
        for window in windows if len(long) else []:
            start = np.maximum(context[long] - window + 1, 0)
            lens_kv = lengths[long] - start
            gather = [block_table[b, np.arange(s, lengths[b]) // c.page_size] * c.page_size
                      + np.arange(s, lengths[b]) % c.page_size for b, s in zip(long, start)]
            narrow.update({f"gather{window}": np.concatenate(gather), f"lens_q{window}": fresh[long],
                           f"lens_kv{window}": lens_kv, f"offsets_q{window}": first[long],
                           f"offsets_kv{window}": np.cumsum(lens_kv) - lens_kv})
        block_heads = sorted({layer.mixer.heads for layer in c.layers if isinstance(layer.mixer, GatedLinearConfig)})
        cut = {}
        if len(long):
            starts = [first[b] + np.arange(0, fresh[b], BLOCK_TOKENS) for b in long]
            narrow["block_rows"] = np.concatenate(starts)
            narrow["block_tokens"] = np.concatenate([np.minimum(first[b] + fresh[b] - start, BLOCK_TOKENS)
                                                     for b, start in zip(long, starts)])
            for heads in block_heads:
                plan = np.asarray(plan_segments([len(start) for start in starts], heads, self.sms))
                narrow[f"segments{heads}"] = np.stack([long[plan[:, 0]], plan[:, 1], plan[:, 2], plan[:, 3]], 1).reshape(-1)
                narrow[f"segment_last{heads}"] = plan[:, 4]
                cut[heads] = bool((plan[:, 4] == 0).any())
        narrow.update({"sequence_of": step.sequence_ids,
                       "row_lens": np.where(fresh[step.sequence_ids] > 0, step.positions + 1, 0)})
        plans = {size: plan_chunks(size, context, fresh, first, long) for size in c.chunks() if len(long)}
        for size, plan in plans.items():
            at = np.asarray(plan["moved"], dtype=np.int64).reshape(-1, 2)
            narrow[f"moved{size}"] = block_table[at[:, 0], at[:, 1] // c.page_size] * c.page_size + at[:, 1] % c.page_size
            narrow.update({f"{name}{size}": plan[name]
                           for name in ("packed", "moved_to", "lens_q", "lens_kv", "offsets_q", "offsets_kv")})
        if c.chunks() and len(long):
            counts = [len(start) for start in starts]
            narrow["whole"] = np.stack([long, np.cumsum(counts) - counts, counts], 1).reshape(-1)
        wide = {"tokens": step.tokens, "pages": step.write_pages, "slots": step.write_slots,
                "query_offsets": step.query_offsets, "page_offsets": step.page_offsets, "page_list": step.pages,
                "last": step.last_page_lengths, "short_rows": short, "positions": step.positions}
        w, n = self._send(wide, np.int64), self._send(narrow, np.int32)
        expanded = {}
        for window in windows if len(long) else []:
            part = lambda name: n[f"{name}{window}"]
            expanded[window] = ExpandedRows(part("gather"), part("gather").numel(), part("lens_q"), part("lens_kv"),
                                            part("offsets_q"), part("offsets_kv"), len(long))
        blocks = {heads: BlockRows(n["block_rows"], n["block_tokens"], n["block_rows"].numel(), n[f"segments{heads}"],
                                   n[f"segment_last{heads}"], n[f"segment_last{heads}"].numel(), cut[heads])
                  for heads in cut}
        chunks = {}
        for size, plan in plans.items():
            part = lambda name: n[f"{name}{size}"]
            chunks[size] = ChunkRows(part("packed"), torch.from_numpy(plan["cached"]).cuda(), plan["keys"], part("moved"),
                                     part("moved_to"), part("lens_q"), part("lens_kv"), part("offsets_q"), part("offsets_kv"),
                                     len(plan["lens_q"]))
        whole = None
        if "whole" in n:
            whole = BlockRows(n["block_rows"], n["block_tokens"], n["block_rows"].numel(), n["whole"], None, len(long), False)
        everything = len(short) == len(step.tokens)
        return StepRows(len(step.tokens), w["tokens"], w["pages"], w["slots"], w["query_offsets"], w["page_offsets"],
                        w["page_list"], w["last"], n["first"], n["fresh"], n["context"],
                        n["table"].view(block_table.shape), w["positions"], n["sequence_of"], n["row_lens"],
                        int(fresh.max()), None if everything else w["short_rows"], n["short_sequences"], n["short_lens"],
                        len(short), expanded, blocks, chunks, whole)

    def _send(self, arrays: dict, kind) -> dict:
        torch = self.torch
        sizes = [len(array) for array in arrays.values()]
        starts = np.cumsum([0] + [round_up(size, 4) for size in sizes])
        packed = np.zeros(int(starts[-1]), dtype=kind)
        for (start, size), array in zip(zip(starts, sizes), arrays.values()):
            packed[start: start + size] = array
        sent = torch.from_numpy(packed).cuda()
        return {name: sent[start: start + size] for name, start, size in zip(arrays, starts, sizes)}


def random_weights(config: HybridConfig, names: dict, seed: int = 4) -> dict:
    """Random bf16 weights on the GPU for ``names`` (name -> shape): matrices ~ N(0, 1 / columns), norms 1, decays that keep a few
    hundred tokens, streams that blend into one another a little."""
    import torch

    generator = torch.Generator(device="cuda").manual_seed(seed)
    constants = {"a2.b": 2.0, "A_log": -3.0, "dt_bias": 0.0, "q.b": 0.0, "k.b": 0.0, "v.b": 0.0}
    weights = {}
    for name, shape in names.items():
        if len(shape) == 1:
            value = next((value for ending, value in constants.items() if name.endswith(ending)), 1.0)
            if name.endswith((".in", ".out")) and ".hc" in name:
                value = 1.0 / shape[0]
            weights[name] = torch.full(shape, value, dtype=torch.bfloat16, device="cuda")
        else:
            values = torch.randn(shape, generator=generator, device="cuda", dtype=torch.float32)
            values *= 1.0 if name == "embed" else shape[1] ** -0.5
            if name.endswith(".mix") and ".hc" in name:
                values = 0.1 * values + torch.eye(shape[0], device="cuda")
            weights[name] = values.to(torch.bfloat16)
    return weights


def decode_step_bytes(config: HybridConfig, sequences: int, context: int) -> dict:
    """Algorithmic HBM bytes of one bf16 decode step: every weight once (borrowed layers read their owner's again), the visible
    latents or keys and values of every sequence, the recurrent states read and written, the residual streams where there are
    several."""
    weights, cache, state, streams = config.vocab * config.width, 0, 0, 0
    for layer in config.layers:
        m, w = layer.mixer, config.width
        weights += (3 if layer.gated else 2) * layer.ffn * w
        streams += sequences * config.streams * w * (2 if layer.ffn else 1)
        if isinstance(m, LatentAttentionConfig):
            weights += (m.q_rank + m.kv_rank + m.heads) * w + m.heads * m.dim * (m.q_rank + m.kv_rank)
            weights += m.heads * m.vdim * (m.kv_rank + w)
            cache += sequences * min(context, m.window) * m.kv_rank
        elif isinstance(m, ParallelConfig):
            a, r = m.left, m.right
            weights += (a.heads * (a.dim + a.vdim) + a.kv_heads * (a.dim + a.vdim)) * w
            weights += (2 * r.kv_heads * r.dim + 2 * r.heads * r.vdim + r.heads + r.rank + r.gate_rank) * w
            weights += r.heads * (r.dim * r.rank + r.vdim * r.gate_rank)
            cache += sequences * (context % a.chunk + 1) * a.kv_heads * (a.dim + a.vdim)
            state += sequences * r.heads * r.dim * r.vdim
        else:
            weights += (2 * m.heads * (m.dim + m.vdim) + m.rank) * w + m.heads * m.dim * m.rank + m.heads * m.vdim * w
            state += sequences * m.heads * m.dim * m.vdim
    total = 2 * weights + 2 * cache + 8 * state + 8 * streams
    return {"weights": 2 * weights, "latents": 2 * cache, "states": 8 * state, "streams": 8 * streams, "total": total}
