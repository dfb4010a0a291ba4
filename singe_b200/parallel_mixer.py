"""Two mixers side by side on the same input, and the two they are:

  ``ChunkedAttention``  grouped-query attention in which a token sees the chunk of positions it stands in.  Projections with
                        biases, a short convolution over time on q, k and v, RMS norm over whole projections, rotation of
                        adjacent pairs (YaRN-scaled frequencies), then attention over the paged cache: the split decode kernel
                        for few tokens, the tensor-core prompt kernel for more, which takes every (sequence, chunk) piece as a
                        sequence of its own.
  ``GatedDelta``        the gated delta rule: short convolutions with silu, unit queries and keys, a recurrent state per
                        sequence, [heads, dim, vdim] in f32, with one decay per key channel; token by token for few tokens,
                        block by block on the tensor core for more.
  ``ParallelMixer``     one projection GEMM for both; their outputs side by side, RMS-normed and averaged by the residual.

Caches and states: keys and values in pages behind the page table; the last projected rows of each sequence for the
convolutions and the recurrent state in the sequence's row, where a sequence's first token starts over, so that a row that is used
again needs no clearing.
"""
from __future__ import annotations

import math
from dataclasses import dataclass

import numpy as np

from . import kernel_sys as ks
from .decoder import PageTable
from .layer_ops import FEW_TOKENS, Ops, StepRows, round_up

TILED_HEAD_SIZES = (64, 128)   # head sizes of the tensor-core kernels; smaller heads are padded with zeros
TILED_GROUP = 8                # most query heads per key/value head of the split decode kernel
TILED_PAGE = 16                # tokens of its pages
NO_WINDOW = 1 << 29
UNIT_EPS = 1e-6                # under the root of a unit vector's squared length


@dataclass(frozen=True)
class YarnScaling:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class Rotation:
    dims: int
    base: float
    scaling: YarnScaling | None = None

    def frequencies(self) -> np.ndarray:
        """Angle per position of each pair of dimensions."""
        index = np.arange(self.dims // 2, dtype=np.float64)
        plain = float(self.base) ** (-2.0 * index / self.dims)
        if self.scaling is None:
            return plain
        s = self.scaling
        # the pair that makes `turns` turns over the original context
        pair = lambda turns: self.dims * math.log(s.original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.base))
        low, high = max(math.floor(pair(s.fast)), 0), min(math.ceil(pair(s.slow)), self.dims - 1)
        ramp = np.clip((index - low) / max(high - low, 0.001), 0.0, 1.0)
        return plain / s.factor * ramp + plain * (1.0 - ramp)

    def magnitude(self) -> float:
        return 1.0 if self.scaling is None else 0.1 * math.log(self.scaling.factor) + 1.0


@dataclass(frozen=True)
class ChunkedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int
    taps: int
    rotation: Rotation


@dataclass(frozen=True)
class GatedDeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    rank: int        # of the decay projection
    gate_rank: int   # of the output gate's projection


@dataclass(frozen=True)
class ParallelConfig:
    left: ChunkedAttentionConfig
    right: GatedDeltaConfig


def side_by_side(ops: Ops, parts, dimension: int = 0):
    """The parts one after the other, each padded with zeros to a multiple of eight."""
    torch = ops.torch
    padded = []
    for part in parts:
        shape = list(part.shape)
        shape[dimension] = round_up(shape[dimension], 8) - shape[dimension]
        padded += [part, torch.zeros(shape, dtype=part.dtype, device=part.device)]
    return torch.cat(padded, dimension).contiguous()


def parts_at(*widths):
    """First columns of parts laid out by ``side_by_side``, and the end."""
    return [0] + [int(end) for end in np.cumsum([round_up(width, 8) for width in widths])]


class ChunkedAttention:
    """Weights of one chunked-attention mixer and its step.  ``source`` maps tensor names to arrays."""

    def __init__(self, config: ChunkedAttentionConfig, source, ops: Ops, eps: float):
        torch = ops.torch
        self.config, self.ops, self.eps = config, ops, eps
        c = config
        take = lambda name: torch.as_tensor(source(name)).to("cuda").to(ops.dtype)
        widest = max(c.dim, c.vdim)
        self.tiled = ops.is_bf16 and widest <= TILED_HEAD_SIZES[-1] and c.heads // c.kv_heads <= TILED_GROUP
        self.size = (next(size for size in TILED_HEAD_SIZES if widest <= size) if self.tiled
                     else round_up(widest, 8 if ops.is_bf16 else 1))
        _, self.key_at, self.value_at, self.span = parts_at(c.heads * c.dim, c.kv_heads * c.dim, c.kv_heads * c.vdim)
        self.inputs = side_by_side(ops, [take("q"), take("k"), take("v")])       # rows of the input projection
        self.bias = side_by_side(ops, [take("q.b"), take("k.b"), take("v.b")])
        self.taps = side_by_side(ops, [take("q.conv").T, take("k.conv").T, take("v.conv").T], 1)
        self.q_norm, self.k_norm = take("q.norm").contiguous(), take("k.norm").contiguous()
        self.frequencies = torch.from_numpy(c.rotation.frequencies()).cuda()
        out = take("o")
        out = torch.nn.functional.pad(out.reshape(out.shape[0], c.heads, c.vdim), (0, self.size - c.vdim))
        self.out = ops.weight(out.reshape(out.shape[0], c.heads * self.size))

    def new_cache(self, table: PageTable, sequences: int):
        torch, c = self.ops.torch, self.config
        zeros = lambda *shape: torch.zeros(shape, dtype=self.ops.dtype, device="cuda")
        pages = (table.page_count(), table.page_size, c.kv_heads, self.size)
        return zeros(*pages), zeros(*pages), zeros(sequences, c.taps - 1, self.span)

    def scratch(self, rows: int, key_bound: int):
        """Partial results of the split decode attention for ``rows`` queries over at most ``key_bound`` keys."""
        if not self.tiled:
            return None
        torch, c = self.ops.torch, self.config
        bound = min(c.chunk + TILED_PAGE - 1, key_bound)
        splits = int(ks.lib().singe_paged_kv_decode_default_splits(rows, c.kv_heads, bound, TILED_PAGE))
        attn = torch.empty((rows, c.heads, splits, self.size), dtype=torch.float32, device="cuda")
        lse = torch.empty((rows, c.heads, splits), dtype=torch.float32, device="cuda")
        return splits, attn, lse

    def attend(self, stream, step: StepRows, projected, cache, out, status, scratch=None) -> None:
        """out = W_o of the heads' outputs; ``projected`` holds this mixer's columns of the input projection."""
        ops, c, size = self.ops, self.config, self.size
        torch = ops.torch
        keys, values, state = cache
        t = projected.shape[0]
        pages, page_size = keys.shape[0], keys.shape[1]
        sequences = step.fresh_tokens.numel()
        buffer = lambda rows, heads: torch.empty((rows, heads * size), dtype=ops.dtype, device="cuda")
        query, attended = buffer(t, c.heads), buffer(t, c.heads)
        rows = step.chunks.get(c.chunk) if self.tiled else None
        packed_keys = packed_values = None
        if rows is not None:
            packed_keys, packed_values = buffer(rows.keys, c.kv_heads), buffer(rows.keys, c.kv_heads)
        conv = [projected, projected.stride(0)]
        ops.call(f"singe_conv_attention_inputs_{ops.suffix}", stream, query, query.stride(0), keys, values, packed_keys,
                 packed_values, *conv, self.bias, self.taps, state, self.q_norm, self.k_norm, self.frequencies,
                 self.frequencies.numel(), c.rotation.magnitude(), step.positions, step.sequence_of, step.first,
                 step.fresh_tokens, step.context, step.pages, step.slots, None if rows is None else rows.cached,
                 None if rows is None else rows.packed, 0 if rows is None else rows.keys, t, sequences, c.taps, c.heads,
                 c.kv_heads, c.dim, c.vdim, size, size, self.key_at, self.value_at, self.span, pages, page_size, self.eps, status)
        if step.longest > 1:
            ops.call(f"singe_conv_state_{ops.suffix}", stream, *conv, state, step.first, step.fresh_tokens, t, sequences, c.taps,
                     self.span)
        if rows is not None:
            self._prompt(stream, rows, query, keys, values, packed_keys, packed_values, attended, status)
        if not self.tiled:
            self._decode(stream, step, query, step.sequence_of, step.row_lens, keys, values, attended, status, None)
        elif step.short_rows is None:
            self._decode(stream, step, query, step.short_sequences, step.short_lens, keys, values, attended, status, scratch)
        elif step.short_count > 0:
            short = buffer(step.short_count, c.heads)
            self._decode(stream, step, query.index_select(0, step.short_rows), step.short_sequences, step.short_lens, keys, values,
                         short, status, scratch)
            attended.index_copy_(0, step.short_rows, short)
        ops.linear(stream, out, attended, self.out)

    def _decode(self, stream, step, query, sequence_of, lens, keys, values, attended, status, scratch) -> None:
        """Every query over the cached keys of its own chunk."""
        ops, c = self.ops, self.config
        sizes = [query.shape[0], c.heads, c.kv_heads, self.size, keys.shape[1], keys.shape[0], step.table.shape[0],
                 step.table.shape[1], c.chunk]
        operands = [query, keys, values, sequence_of, lens, step.table]
        if not ops.is_bf16:
            ops.call("singe_chunked_attention_f32", stream, attended, *operands, *sizes, c.scale, status)
            return
        splits, attn, lse = scratch or self.scratch(query.shape[0], step.table.shape[1] * keys.shape[1]) or (1, None, None)
        ops.call("singe_chunked_attention_bf16", stream, attended, attn, lse, *operands, *sizes, splits, c.scale, status)

    def _prompt(self, stream, rows, query, keys, values, packed_keys, packed_values, attended, status) -> None:
        ops, c, size = self.ops, self.config, self.size
        width = c.kv_heads * size
        if rows.moved.numel() > 0:
            for packed, cache in ((packed_keys, keys), (packed_values, values)):
                ops.call("singe_move_rows", stream, packed, cache, rows.moved, rows.moved_to, rows.moved.numel(), width * 2,
                         cache.shape[0] * cache.shape[1], rows.keys, status)
        lse = ops.torch.empty((query.shape[0], c.heads), dtype=ops.torch.float32, device="cuda")
        ops.call("singe_windowed_prefill_attention_bf16", stream, attended, lse, query, packed_keys, packed_values, width,
                 rows.lens_q, rows.lens_kv, rows.offsets_q, rows.offsets_kv, None, 0, rows.pieces, query.shape[0], rows.keys,
                 c.heads, c.kv_heads, size, NO_WINDOW, c.scale)


class GatedDelta:
    """Weights of one gated-delta mixer and its step.  ``source`` maps tensor names to arrays."""

    def __init__(self, config: GatedDeltaConfig, source, ops: Ops, eps: float):
        torch = ops.torch
        self.config, self.ops, self.eps = config, ops, eps
        c = config
        take = lambda name: torch.as_tensor(source(name)).to("cuda").to(ops.dtype)
        _, self.key_at, self.value_at, self.span = parts_at(c.kv_heads * c.dim, c.kv_heads * c.dim, c.heads * c.vdim)
        self.rank = round_up(max(c.rank, c.gate_rank), 8)
        self.strength_at = self.span
        self.low_at = self.strength_at + round_up(c.heads, 8)
        pad = torch.nn.functional.pad
        low = [pad(take(name), (0, 0, 0, self.rank - rank)) for name, rank in (("a1", c.rank), ("g1", c.gate_rank))]
        self.inputs = side_by_side(ops, [take("q"), take("k"), take("v"), take("b"), *low])
        self.taps = side_by_side(ops, [take("q.conv").T, take("k.conv").T, take("v.conv").T], 1)
        # the second halves of the two low-rank projections, as a product of two "heads"
        self.columns = round_up(max(c.heads * c.dim, c.heads * c.vdim), 8)
        self.second = torch.stack([pad(take(name), (0, self.rank - rank, 0, self.columns - size))
                                   for name, rank, size in (("a2", c.rank, c.heads * c.dim), ("g2", c.gate_rank, c.heads * c.vdim))]
                                  ).contiguous()
        self.decay_rate, self.decay_bias = ops.scalars(source("A_log")), ops.scalars(source("dt_bias"))
        self.norm = take("norm").contiguous()
        self.out = ops.weight(take("o"))
        # the block form, for sizes it takes
        self.blocked = ops.is_bf16 and ks.lib().singe_gated_delta_prompt_scratch(c.heads, c.dim, c.vdim, 1, 1) > 0

    def new_cache(self, table: PageTable, sequences: int):
        torch, c = self.ops.torch, self.config
        return (torch.zeros((sequences, c.heads, c.dim, c.vdim), dtype=torch.float32, device="cuda"),
                torch.zeros((sequences, c.taps - 1, self.span), dtype=self.ops.dtype, device="cuda"))

    def attend(self, stream, step: StepRows, projected, cache, out, status, scratch=None) -> None:
        """out = W_o of the heads' outputs; ``projected`` holds this mixer's columns of the input projection."""
        ops, c = self.ops, self.config
        torch = ops.torch
        state, conv_state = cache
        t, sequences = projected.shape[0], state.shape[0]
        mixed = ops.rows(t, self.span)
        inverse = torch.empty((t, 2 * c.kv_heads), dtype=torch.float32, device="cuda")
        conv = [projected, projected.stride(0)]
        ops.call(f"singe_conv_recurrence_inputs_{ops.suffix}", stream, mixed, mixed.stride(0), inverse, *conv, self.taps, conv_state,
                 step.sequence_of, step.first, step.fresh_tokens, step.context, t, sequences, c.taps, c.kv_heads, c.dim, self.key_at,
                 self.span, UNIT_EPS)
        if step.longest > 1:
            ops.call(f"singe_conv_state_{ops.suffix}", stream, *conv, conv_state, step.first, step.fresh_tokens, t, sequences, c.taps,
                     self.span)
        decay = ops.rows(t, 2 * self.columns)
        ops.head_linear(stream, decay, projected[:, self.low_at: self.low_at + 2 * self.rank], self.second, 2)
        attended = ops.rows(t, c.heads * c.vdim)
        strength = projected[:, self.strength_at:]
        operands = [attended, attended.stride(0), mixed, mixed.stride(0), inverse, strength, strength.stride(0), decay,
                    decay.stride(0), self.decay_rate, self.decay_bias, self.norm, state]
        sizes = [c.heads, c.kv_heads, c.dim, c.vdim, self.key_at, self.value_at, self.columns, self.eps]
        rows = step.whole if self.blocked else None
        if rows is not None:
            scratch = torch.empty(int(ks.lib().singe_gated_delta_prompt_scratch(c.heads, c.dim, c.vdim, t, rows.blocks)),
                                  dtype=torch.uint8, device="cuda")
            ops.call("singe_gated_delta_prompt_bf16", stream, *operands, step.context, t, *sizes, rows.rows, rows.tokens, rows.blocks,
                     rows.segments, rows.count, scratch)
        if rows is None or step.short_count > 0:
            ops.call(f"singe_gated_delta_step_{ops.suffix}", stream, *operands, step.first, step.fresh_tokens, step.context, t,
                     sequences, *sizes, 0x7fffffff if rows is None else FEW_TOKENS)
        ops.linear(stream, out, attended, self.out)


class ParallelMixer:
    """Both sides of a layer and its step.  The two outputs stand side by side in ``delta``, the right one from a multiple of
    eight columns on; ``output_norms`` are the weights of their norms."""

    def __init__(self, config: ParallelConfig, source, ops: Ops, eps: float):
        self.config, self.ops = config, ops
        self.left = ChunkedAttention(config.left, lambda name: source("left." + name), ops, eps)
        self.right = GatedDelta(config.right, lambda name: source("right." + name), ops, eps)
        self.project = ops.weight(ops.torch.cat([self.left.inputs, self.right.inputs]))
        self.split = self.left.inputs.shape[0]
        self.left.inputs = self.right.inputs = None
        self.output_norms = (ops.weight(source("left.out")), ops.weight(source("right.out")))

    def new_cache(self, table: PageTable, sequences: int):
        return self.left.new_cache(table, sequences) + self.right.new_cache(table, sequences)

    def scratch(self, rows: int, key_bound: int):
        return self.left.scratch(rows, key_bound)

    def run(self, stream, step: StepRows, normed, cache, delta, status, scratch=None) -> None:
        projected = self.ops.rows(normed.shape[0], self.project.shape[0])
        self.ops.linear(stream, projected, normed, self.project)
        width = normed.shape[1]
        right = delta.shape[1] - width
        self.left.attend(stream, step, projected[:, :self.split], cache[:3], delta[:, :width], status, scratch)
        self.right.attend(stream, step, projected[:, self.split:], cache[3:], delta[:, right:], status)
