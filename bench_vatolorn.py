"""The Vatolorn decoder beside Kavalorn and the Llama-shaped decoder at equal size: decode and prompt throughput of six layers
each, and its kernels beside their like kernels against their rooflines.  ``python bench.py --model vatolorn`` prints the figures
as one JSON line.  Random bf16 weights and token ids; device time by CUDA events.
"""
from __future__ import annotations

import math

import numpy as np
import torch

import bench_hybrid as peer_bench
from bench_extra import graph_seconds, rotating
from bench_hybrid import _compute, _memory, _stream, decode_figures, hybrid_decoder, normal, prompt_figures
from singe_b200 import checkpoint, hybrid, kernel_sys as ks, llama
from singe_b200.parallel_mixer import (TILED_PAGE, ChunkedAttentionConfig, GatedDeltaConfig, ParallelConfig, Rotation,
                                       YarnScaling)

# name -> (width, heads, kv heads, head size, chunk, recurrent heads, their q/k heads, key size, value size, rank, ffn, vocab);
# heads, head size, width, ffn and vocabulary as the other decoders of this name have them
SIZES = {
    "2048": (2048, 16, 4, 128, 4096, 16, 16, 64, 128, 64, 8192, 32000),
    "4096": (4096, 32, 8, 128, 8192, 32, 16, 128, 128, 128, 14336, 128256),
}
LAYERS, STREAMS, TAPS = 6, 4, 4


def config_of(size: str) -> hybrid.HybridConfig:
    width, heads, kv, dim, chunk, r_heads, r_kv, key, value, rank, ffn, vocab = SIZES[size]
    mixer = ParallelConfig(
        ChunkedAttentionConfig(heads, kv, dim, dim, dim ** -0.5, chunk, TAPS, Rotation(dim, 10000.0, YarnScaling(8.0, 4096.0, 32.0, 1.0))),
        GatedDeltaConfig(r_heads, r_kv, key, value, TAPS, rank, rank))
    return hybrid.HybridConfig(layers=[hybrid.LayerConfig(mixer, ffn, None, True)] * LAYERS, width=width, vocab=vocab, page_size=TILED_PAGE,
                               streams=STREAMS, logit_scale=0.5)


def model_figures(size: str, peaks) -> dict:
    ours, kavalorn, peer = config_of(size), peer_bench.hybrid_config(size), peer_bench.llama_config(size, LAYERS)
    flops = lambda config: 2.0 * sum(math.prod(shape) for name, shape in checkpoint.hybrid_names(config).items()
                                     if len(shape) == 2 and name not in ("embed", "head") and not name.endswith(".conv"))
    kv = (peer.heads + 2 * peer.kv_heads) * peer.head_dim
    peer_flops = 2.0 * peer.layers * (peer.hidden * kv + peer.heads * peer.head_dim * peer.hidden + 3 * peer.hidden * peer.ffn)
    models = {"vatolorn": (lambda s, c: hybrid_decoder(ours, s, c), lambda s, c: hybrid.decode_step_bytes(ours, s, c)["total"], flops(ours)),
              "kavalorn": (lambda s, c: hybrid_decoder(kavalorn, s, c), lambda s, c: hybrid.decode_step_bytes(kavalorn, s, c)["total"],
                           flops(kavalorn)),
              "llama": (lambda s, c: llama.LlamaDecoder(peer, s, c), lambda s, c: llama.decode_step_bytes(peer, s, c)["total"], peer_flops)}
    out = {}
    for sequences, context in ((64, 2048), (8, 8190)):
        row = out[f"decode {sequences} x {context}"] = {}
        for name, (make, moved, _) in models.items():
            row[name] = decode_figures(make, moved(sequences, context), sequences, context, ours.vocab, peaks)
            torch.cuda.empty_cache()
    for lengths in ([8192], [2048] * 4, [480, 240, 120, 60] * 16):
        key = f"prompt {len(lengths)} x {lengths[0]}" if len(set(lengths)) == 1 else f"prompt {len(lengths)} of {lengths[:4]}"
        row = out[key] = {}
        for name, (make, _, linear) in models.items():
            row[name] = prompt_figures(make, lengths, ours.vocab, linear, peaks)
            torch.cuda.empty_cache()
    return out


# ------------------------------------------------------------------------------------------------
# kernels
# ------------------------------------------------------------------------------------------------

def decode_attention(size: str, sequences: int, visible: int, peaks) -> dict:
    """The chunked decode attention with ``visible`` keys of the current chunk behind as many hidden ones."""
    _, heads, kv, dim, *_ = SIZES[size]
    o = hybrid.Ops("bfloat16")
    stride = -(-2 * visible // TILED_PAGE)
    splits = int(ks.lib().singe_paged_kv_decode_default_splits(sequences, kv, visible + TILED_PAGE - 1, TILED_PAGE))
    attn, lse = torch.empty((sequences, heads, splits, dim), device="cuda"), torch.empty((sequences, heads, splits), device="cuda")
    order, lens = torch.arange(sequences, dtype=torch.int32, device="cuda"), torch.full((sequences,), 2 * visible, dtype=torch.int32, device="cuda")
    status = torch.zeros(1, dtype=torch.int32, device="cuda")

    def make(i):
        keys, values = normal(sequences * stride, TILED_PAGE, kv, dim), normal(sequences * stride, TILED_PAGE, kv, dim)
        table = torch.randperm(sequences * stride, device="cuda").to(torch.int32).view(sequences, stride)
        query, out = normal(sequences, heads, dim), torch.empty((sequences, heads, dim), dtype=torch.bfloat16, device="cuda")
        return lambda: o.call("singe_chunked_attention_bf16", _stream(), out, attn, lse, query, keys, values, order, lens, table, sequences,
                              heads, kv, dim, TILED_PAGE, sequences * stride, sequences, stride, visible, splits, dim ** -0.5, status)

    moved = sequences * visible * kv * dim * 4
    call, _ = rotating(make, moved)
    return {"shape": f"{sequences} x {visible} keys, {heads} heads on {kv}, {splits} splits", **_memory(graph_seconds(call), moved, peaks)}


def prompt_attention(size: str, lengths, peaks) -> dict:
    _, heads, kv, dim, chunk, *_ = SIZES[size]
    o, total = hybrid.Ops("bfloat16"), sum(lengths)
    pieces = [min(chunk, n - at) for n in lengths for at in range(0, n, chunk)]
    query, out = normal(total, heads, dim), torch.empty((total, heads, dim), dtype=torch.bfloat16, device="cuda")
    keys, values, lse = normal(total, kv, dim), normal(total, kv, dim), torch.empty((total, heads), device="cuda")
    lens = torch.tensor(pieces, dtype=torch.int32, device="cuda")
    offsets = torch.tensor(np.cumsum([0] + pieces)[:-1], dtype=torch.int32, device="cuda")
    call = lambda: o.call("singe_windowed_prefill_attention_bf16", _stream(), out, lse, query, keys, values, kv * dim, lens, lens, offsets,
                          offsets, None, 0, len(pieces), total, total, heads, kv, dim, 1 << 29, dim ** -0.5)
    flops = 4.0 * heads * dim * sum(n * (n + 1) / 2 for n in pieces)
    return {"shape": f"{len(lengths)} x {lengths[0]} tokens in pieces of {pieces[0]}, {heads} heads of {dim} on {kv}",
            **_compute(graph_seconds(call, 4), flops, peaks)}


class DeltaOperands:
    """Random operands of the recurrence kernels for ``rows`` tokens; decays that keep a few hundred tokens."""

    def __init__(self, size: str, rows: int, sequences: int):
        _, _, _, _, _, heads, kv, key, value, *_ = SIZES[size]
        o = self.o = hybrid.Ops("bfloat16")
        self.heads, self.kv, self.key, self.value = heads, kv, key, value
        self.key_at, self.value_at, self.columns = kv * key, 2 * kv * key, heads * max(key, value)
        self.mixed, self.decay, self.strength = o.rows(rows, self.value_at + heads * value), o.rows(rows, 2 * self.columns), normal(rows, heads)
        self.mixed.normal_()
        self.decay.normal_()
        self.inverse = torch.full((rows, 2 * kv), key ** -0.5, device="cuda")
        self.rate, self.bias = torch.full((heads,), -3.0, device="cuda"), torch.zeros(heads * key, device="cuda")
        self.norm, self.out = normal(value), o.rows(rows, heads * value)
        self.state = normal(sequences, heads, key, value, kind=torch.float32)
        self.operands = [self.out, self.out.stride(0), self.mixed, self.mixed.stride(0), self.inverse, self.strength, heads, self.decay,
                         self.decay.stride(0), self.rate, self.bias, self.norm, self.state]
        self.sizes = [heads, kv, key, value, self.key_at, self.value_at, self.columns, 1e-6]
        # every operand of a token once: q, k, v, z, gate, b in; out
        self.token_bytes = 2 * (self.value_at + heads * value + heads * key + heads * value + heads) + 2 * heads * value


def recurrence_step(size: str, sequences: int, peaks) -> dict:
    one, first = torch.ones(sequences, dtype=torch.int32, device="cuda"), torch.arange(sequences, dtype=torch.int32, device="cuda")

    def make(i):
        d = DeltaOperands(size, sequences, sequences)
        return lambda: d.o.call("singe_gated_delta_step_bf16", _stream(), *d.operands, first, one, one, sequences, sequences, *d.sizes, 8)

    d = DeltaOperands(size, sequences, sequences)
    moved = sequences * (8 * d.heads * d.key * d.value + d.token_bytes)
    call, _ = rotating(make, moved)
    return {"shape": f"{sequences} x {d.heads} heads, state {d.key} x {d.value}", **_memory(graph_seconds(call), moved, peaks)}


def recurrence_prompt(size: str, lengths, peaks) -> dict:
    total = sum(lengths)
    d = DeltaOperands(size, total, len(lengths))
    i32 = lambda a: torch.tensor(np.ascontiguousarray(a), dtype=torch.int32, device="cuda")
    firsts = np.cumsum([0] + lengths)[:-1]
    starts = [np.arange(f, f + n, 16) for f, n in zip(firsts, lengths)]
    tokens = np.concatenate([np.minimum(f + n - s, 16) for f, n, s in zip(firsts, lengths, starts)])
    counts = [len(s) for s in starts]
    rows, tokens = i32(np.concatenate(starts)), i32(tokens)
    runs = i32(np.stack([np.arange(len(lengths)), np.cumsum(counts) - counts, counts], 1))
    context = torch.zeros(len(lengths), dtype=torch.int32, device="cuda")
    scratch = torch.empty(int(ks.lib().singe_gated_delta_prompt_scratch(d.heads, d.key, d.value, total, rows.numel())), dtype=torch.uint8,
                          device="cuda")
    call = lambda: d.o.call("singe_gated_delta_prompt_bf16", _stream(), *d.operands, context, total, *d.sizes, rows, tokens, rows.numel(), runs,
                            len(lengths), scratch)
    return {"shape": f"{len(lengths)} x {lengths[0]} tokens, {d.heads} heads, state {d.key} x {d.value}",
            **_memory(graph_seconds(call, 4), total * d.token_bytes, peaks)}


def glue_kernels(size: str, rows: int, peaks) -> dict:
    """One sequence per row for a decode batch, one sequence for a prompt."""
    width, heads, kv, dim, _, r_heads, r_kv, key, value, rank, *_ = SIZES[size]
    o = hybrid.Ops("bfloat16")
    decode = rows <= 128
    i32 = lambda a: torch.tensor(a, dtype=torch.int32, device="cuda")
    sequences = rows if decode else 1
    sequence_of = torch.arange(rows, dtype=torch.int32, device="cuda") if decode else torch.zeros(rows, dtype=torch.int32, device="cuda")
    first, fresh, context = (sequence_of, i32([1] * rows), i32([9] * rows)) if decode else (i32([0]), i32([rows]), i32([0]))

    def streams(parts):
        def make(i):
            x, delta, normed = torch.randn((rows, STREAMS, width), device="cuda"), normal(rows, parts * width), o.rows(rows, width)
            gains, blend, weight = normal(2, width), torch.eye(STREAMS, device="cuda"), normal(width)
            ones = torch.full((STREAMS,), 0.25, device="cuda")
            return lambda: o.call("singe_stream_step_norm_bf16", _stream(), x, delta, parts * width, parts, width, gains[0], gains[1], 0.5, blend,
                                  ones, ones, 1, normed, width, weight, 1.0, rows, STREAMS, width, 1e-6)

        return make, rows * width * (8 * STREAMS + 2 * parts + 2)

    attention_span, delta_span = (heads + 2 * kv) * dim, 2 * r_kv * key + r_heads * value

    def attention_inputs():
        def make(i):
            projected, query = normal(rows, attention_span), normal(rows, heads * dim)
            keys, values = normal(-(-rows // 16), 16, kv, dim), normal(-(-rows // 16), 16, kv, dim)
            index = torch.arange(rows, device="cuda")
            pages, slots, bias, taps = index // 16, index % 16, normal(attention_span), normal(TAPS, attention_span)
            state, qn, kn = normal(sequences, TAPS - 1, attention_span), normal(heads * dim), normal(kv * dim)
            frequencies = torch.rand(dim // 2, dtype=torch.float64, device="cuda")
            return lambda: o.call("singe_conv_attention_inputs_bf16", _stream(), query, heads * dim, keys, values, None, None, projected,
                                  attention_span, bias, taps, state, qn, kn, frequencies, dim // 2, 1.2, index, sequence_of, first, fresh, context,
                                  pages, slots, None, None, 0, rows, sequences, TAPS, heads, kv, dim, dim, dim, dim, heads * dim,
                                  (heads + kv) * dim, attention_span, keys.shape[0], 16, 1e-6, None)

        return make, 2 * (2 * rows + (2 * (TAPS - 1) * rows if decode else 0)) * attention_span

    def recurrence_inputs():
        def make(i):
            projected, mixed, taps = normal(rows, delta_span), o.rows(rows, delta_span), normal(TAPS, delta_span)
            state, inverse = normal(sequences, TAPS - 1, delta_span), torch.empty((rows, 2 * r_kv), device="cuda")
            return lambda: o.call("singe_conv_recurrence_inputs_bf16", _stream(), mixed, mixed.stride(0), inverse, projected, delta_span, taps,
                                  state, sequence_of, first, fresh, context, rows, sequences, TAPS, r_kv, key, r_kv * key, delta_span, 1e-6)

        return make, 2 * (2 * rows + (2 * (TAPS - 1) * rows if decode else 0)) * delta_span

    out = {}
    for name, (make, moved) in (("streams + two normed outputs", streams(2)), ("streams + one output", streams(1)),
                                ("convolution, norms, rotation, cache write", attention_inputs()),
                                ("convolution, silu, unit lengths", recurrence_inputs())):
        call, _ = rotating(make, moved)
        out[name] = _memory(graph_seconds(call), moved, peaks)
    return out


def linear_kernels(size: str, rows: int, peaks) -> dict:
    width, heads, kv, dim, _, r_heads, r_kv, key, value, rank, ffn, _ = SIZES[size]
    o = hybrid.Ops("bfloat16")
    inputs = (heads + 2 * kv) * dim + 2 * r_kv * key + r_heads * value + r_heads + 2 * rank
    out = {}
    for name, (n, k, activation) in {"both mixers in": (inputs, width, 0), "attention out": (width, heads * dim, 0),
                                     "recurrence out": (width, r_heads * value, 0), "gate/up + swiglu": (2 * ffn, width, 1),
                                     "down": (width, ffn, 0)}.items():
        x, y = normal(rows, k), o.rows(rows, n // 2 if activation == 1 else n)

        def make(i):
            w = normal(n, k, scale=k ** -0.5)
            return lambda: o.linear(_stream(), y, x, w, activation)

        if rows <= 128:
            call, _ = rotating(make, n * k * 2)
            out[name] = {"shape": f"{rows} x {n} x {k}", **_memory(graph_seconds(call), 2 * (n * k + rows * (n + k)), peaks)}
        else:
            out[name] = {"shape": f"{rows} x {n} x {k}", **_compute(graph_seconds(make(0), 4), 2.0 * rows * n * k, peaks)}
    columns, x = r_heads * max(key, value), normal(rows, 2 * rank)
    y = o.rows(rows, 2 * columns)

    def make(i):
        w = normal(2, columns, rank)
        return lambda: o.head_linear(_stream(), y, x, w, 2)

    moved = 2 * 2 * (columns * rank + rows * (columns + rank))
    call, _ = rotating(make, moved)
    out["low-rank second halves"] = {"shape": f"2 x ({rows} x {columns} x {rank})", **_memory(graph_seconds(call), moved, peaks)}
    return out


def kernel_figures(size: str, peaks) -> dict:
    torch.manual_seed(0)
    p = peer_bench
    out = {"decode attention": {f"{s} x {c}": {"vatolorn": decode_attention(size, s, c, peaks), "llama": p.paged_decode_kernel(size, s, c, peaks)}
                                for s, c in ((64, 2048), (8, 4096), (64, 512))},
           "prompt attention": {f"{len(l)} x {l[0]}": {"vatolorn": prompt_attention(size, l, peaks),
                                                       "llama": p.prompt_attention_kernels(size, l, peaks)["llama"]}
                                for l in ([8192], [2048] * 4, [512] * 16)},
           "recurrence, one token": {str(s): {"vatolorn": recurrence_step(size, s, peaks), "kavalorn": p.recurrence_step_kernel(size, s, peaks)}
                                     for s in (64, 8)},
           "recurrence, prompt": {f"{len(l)} x {l[0]}": {"vatolorn": recurrence_prompt(size, l, peaks),
                                                         "kavalorn": p.recurrence_prompt_kernel(size, l, peaks)}
                                  for l in ([8192], [2048] * 4, [512] * 16)}}
    for rows in (64, 8192):
        out[f"glue, {rows} rows"] = {"vatolorn": glue_kernels(size, rows, peaks), "others": p.glue_kernels(size, rows, peaks)}
        out[f"linears, {rows} rows"] = {"vatolorn": linear_kernels(size, rows, peaks), "others": p.linear_kernels(size, rows, peaks)}
    torch.cuda.empty_cache()
    return out


def run(peaks, sizes=tuple(SIZES), parts=("model", "kernels")) -> dict:
    out = {}
    for size in sizes:
        out[size] = {}
        if "kernels" in parts:
            out[size]["kernels"] = kernel_figures(size, peaks)
        if "model" in parts:
            out[size]["model"] = model_figures(size, peaks)
    return out
