"""The layer-list decoder (Kavalorn) beside the Llama-shaped decoder at equal size: decode and prompt throughput of a few
layers each, and the kernels of both against their rooflines.  ``python bench.py --model kavalorn`` prints the figures as
one JSON line.  Random bf16 weights and token ids; device time by CUDA events.
"""
from __future__ import annotations

import math

import numpy as np
import torch

from bench_extra import graph_seconds, rotating
from singe_b200 import checkpoint, hybrid, llama, ops

# name -> (width, heads, head size, query latent, key/value latent, window, ffn, recurrent heads, key size, value size, vocab)
SIZES = {
    "2048": (2048, 16, 128, 768, 256, 1024, 8192, 16, 64, 128, 32000),
    "4096": (4096, 32, 128, 1536, 512, 4096, 14336, 32, 64, 128, 128256),
}
PAGE = hybrid.HybridConfig().page_size
PATTERN = "aagaag"   # a: latent attention and feed-forward; g: gated linear attention and feed-forward


def hybrid_config(size: str, pattern: str = PATTERN) -> hybrid.HybridConfig:
    width, heads, dim, q_rank, kv_rank, window, ffn, gla_heads, key, value, vocab = SIZES[size]
    attention = hybrid.LatentAttentionConfig(heads, dim, dim, q_rank, kv_rank, dim ** -0.5, window)
    recurrent = hybrid.GatedLinearConfig(gla_heads, key, value, 16, 16.0)
    layers = [hybrid.LayerConfig(attention if kind == "a" else recurrent, ffn) for kind in pattern]
    return hybrid.HybridConfig(layers=layers, width=width, vocab=vocab)


def hybrid_decoder(config, sequences: int, capacity: int) -> hybrid.HybridDecoder:
    """A layer-list decoder with random weights."""
    weights = hybrid.random_weights(config, checkpoint.hybrid_names(config))
    return hybrid.HybridDecoder(config, sequences, capacity, weights)


def llama_config(size: str, layers: int) -> llama.LlamaConfig:
    width, heads, dim, _, _, _, ffn, _, _, _, vocab = SIZES[size]
    return llama.LlamaConfig(layers=layers, hidden=width, heads=heads, kv_heads=heads // 4, head_dim=dim, ffn=ffn, vocab=vocab)


def decode_figures(make, bytes_per_step: int, sequences: int, context: int, vocab: int, peaks, steps: int = 20) -> dict:
    decoder = make(sequences, context + 64)
    decoder.fill_context(context)
    tokens = np.random.default_rng(4).integers(0, vocab, size=sequences)
    decoder.capture()
    decoder.plan(tokens)
    for _ in range(3):
        decoder.run()
    begin, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    begin.record()
    for _ in range(steps):
        decoder.run()
    end.record()
    torch.cuda.synchronize()
    seconds = begin.elapsed_time(end) * 1e-3 / steps
    assert int(decoder.status.item()) == 0
    return {"ms_per_step": round(seconds * 1e3, 4), "tokens_per_s": round(sequences / seconds, 1),
            "gb_per_step": round(bytes_per_step / 1e9, 3), "frac_hbm": round(bytes_per_step / seconds / 1e9 / peaks["hbm_gbs"], 3)}


def prompt_figures(make, lengths, vocab: int, linear_flops: float, peaks) -> dict:
    decoder = make(len(lengths), max(lengths) + 16)
    rng = np.random.default_rng(5)
    prompts = [rng.integers(0, vocab, size=n).tolist() for n in lengths]
    best = float("inf")
    for _ in range(4):
        decoder.reset()
        torch.cuda.synchronize()
        begin, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        begin.record()
        decoder.step_tokens(prompts)
        end.record()
        torch.cuda.synchronize()
        best = min(best, begin.elapsed_time(end) * 1e-3)
    assert int(decoder.status.item()) == 0
    total = sum(lengths)
    return {"tokens": total, "ms": round(best * 1e3, 3), "tokens_per_s": round(total / best, 1),
            "linear_tflops": round(linear_flops * total / best / 1e12, 1),
            "timing": "CUDA events around one step, the host's planning of it included"}


def model_figures(size: str, peaks) -> dict:
    config = hybrid_config(size)
    names = checkpoint.hybrid_names(config)
    peer = llama_config(size, len(config.layers))
    make = lambda sequences, capacity: hybrid_decoder(config, sequences, capacity)
    make_peer = lambda sequences, capacity: llama.LlamaDecoder(peer, sequences, capacity)
    kv = (peer.heads + 2 * peer.kv_heads) * peer.head_dim
    peer_flops = 2.0 * peer.layers * (peer.hidden * kv + peer.heads * peer.head_dim * peer.hidden + 3 * peer.hidden * peer.ffn)
    flops = 2.0 * sum(math.prod(shape) for name, shape in names.items() if len(shape) == 2 and name not in ("embed", "head"))
    out = {}
    for sequences, context in ((64, 2048), (8, 8192)):
        key = f"decode {sequences} x {context}"
        out[key] = {"kavalorn": decode_figures(make, hybrid.decode_step_bytes(config, sequences, context)["total"], sequences,
                                               context, config.vocab, peaks),
                    "llama": decode_figures(make_peer, llama.decode_step_bytes(peer, sequences, context)["total"], sequences,
                                            context, peer.vocab, peaks)}
        torch.cuda.empty_cache()
    for lengths in ([8192], [2048] * 4, [480, 240, 120, 60] * 16):
        key = f"prompt {len(lengths)} x {lengths[0]}" if len(set(lengths)) == 1 else f"prompt {len(lengths)} of {lengths[:4]}"
        out[key] = {"kavalorn": prompt_figures(make, lengths, config.vocab, flops, peaks),
                    "llama": prompt_figures(make_peer, lengths, peer.vocab, peer_flops, peaks)}
        torch.cuda.empty_cache()
    return out


# ------------------------------------------------------------------------------------------------
# kernels
# ------------------------------------------------------------------------------------------------

def _stream():
    return int(torch.cuda.current_stream().cuda_stream)


def _memory(seconds: float, moved: float, peaks) -> dict:
    return {"us": round(seconds * 1e6, 2), "gbs": round(moved / seconds / 1e9, 1),
            "frac": round(moved / seconds / 1e9 / peaks["hbm_gbs"], 3), "bound": "hbm"}


def _compute(seconds: float, flops: float, peaks) -> dict:
    return {"us": round(seconds * 1e6, 2), "tflops": round(flops / seconds / 1e12, 1),
            "frac": round(flops / seconds / 1e12 / peaks["bf16_tflops"], 3), "bound": "bf16"}


def normal(*shape, scale=1.0, kind=torch.bfloat16):
    return (torch.randn(shape, device="cuda") * scale).to(kind)


def latent_decode_kernel(size: str, sequences: int, context: int, peaks) -> dict:
    _, heads, _, _, latent, window, *_ = SIZES[size]
    o = hybrid.Ops("bfloat16")
    stride = -(-context // PAGE)
    from singe_b200 import kernel_sys as ks

    seen = min(context, window)
    splits = int(ks.lib().singe_latent_decode_splits(sequences, heads, latent, seen))
    attn = torch.empty((sequences, splits, heads, latent), device="cuda")
    lse = torch.empty((sequences, splits, heads), device="cuda")
    order = torch.arange(sequences, dtype=torch.int32, device="cuda")
    lens = torch.full((sequences,), context, dtype=torch.int32, device="cuda")
    status = torch.zeros(1, dtype=torch.int32, device="cuda")

    def make(i):
        cache = normal(sequences * stride, PAGE, latent)
        table = torch.randperm(sequences * stride, device="cuda").to(torch.int32).view(sequences, stride)
        query, out = normal(sequences, heads, latent), torch.empty((sequences, heads, latent), dtype=torch.bfloat16, device="cuda")
        return lambda: o.call("singe_latent_decode_bf16", _stream(), out, attn, lse, query, cache, order, lens, table, sequences,
                              heads, latent, PAGE, sequences * stride, sequences, stride, window, splits, latent ** -0.5, status)

    moved = sequences * (seen + 2 * heads) * latent * 2
    call, _ = rotating(make, moved)
    return {"shape": f"{sequences} x {seen} keys, {heads} heads, latent {latent}, {splits} splits", **_memory(graph_seconds(call), moved, peaks)}


def paged_decode_kernel(size: str, sequences: int, context: int, peaks) -> dict:
    _, heads, dim, *_ = SIZES[size]
    kv = heads // 4
    stride = -(-context // 16)
    config = ops.PagedKvDecodeAttentionConfig.contiguous(sequences, heads, kv, dim, 16, sequences * stride, stride, dim ** -0.5)
    lens = torch.full((sequences,), context, dtype=torch.int32, device="cuda")

    def make(i):
        keys, values = normal(sequences * stride, 16, kv, dim), normal(sequences * stride, 16, kv, dim)
        table = torch.randperm(sequences * stride, device="cuda").to(torch.int32).view(sequences, stride)
        query, out = normal(sequences, heads, dim), torch.empty((sequences, heads, dim), dtype=torch.bfloat16, device="cuda")
        return lambda: ops.paged_kv_decode_attention(out, query, keys, values, lens, table, config)

    moved = sequences * context * kv * dim * 4
    call, _ = rotating(make, moved)
    return {"shape": f"{sequences} x {context} keys, {heads} heads on {kv}", **_memory(graph_seconds(call), moved, peaks)}


def prompt_attention_kernels(size: str, lengths, peaks) -> dict:
    _, heads, dim, _, _, window, *_ = SIZES[size]
    total = sum(lengths)
    o = hybrid.Ops("bfloat16")
    query, gate, out = normal(total, heads, dim), normal(total, heads), torch.empty((total, heads, dim), dtype=torch.bfloat16, device="cuda")
    rows = normal(total, 2, heads, dim)
    lse = torch.empty((total, heads), device="cuda")
    lens = torch.tensor(lengths, dtype=torch.int32, device="cuda")
    offsets = torch.tensor(np.cumsum([0] + lengths)[:-1], dtype=torch.int32, device="cuda")
    windowed = lambda: o.call("singe_windowed_prefill_attention_bf16", _stream(), out, lse, query, rows, rows.data_ptr() + heads * dim * 2,
                              2 * heads * dim, lens, lens, offsets, offsets, gate, heads, len(lengths), total, total, heads, heads, dim,
                              window, dim ** -0.5)
    kv = heads // 4
    keys, values = normal(total, kv, dim), normal(total, kv, dim)
    config = ops.RaggedKvPrefillAttentionConfig(len(lengths), total, total, heads, kv, dim, True, dim ** -0.5)
    causal = lambda: ops.ragged_kv_prefill_attention(out, lse, query, keys, values, lens, lens, offsets, config)
    seen = lambda w: sum(min(i + 1, w) for n in lengths for i in range(n))
    flops = lambda w: 4.0 * heads * dim * seen(w)
    shape = f"{len(lengths)} x {lengths[0]} tokens, {heads} heads of {dim}"
    return {"kavalorn": {"shape": f"{shape}, window {window}", **_compute(graph_seconds(windowed, 4), flops(window), peaks)},
            "llama": {"shape": f"{shape} on {kv}", **_compute(graph_seconds(causal, 4), flops(1 << 30), peaks)}}


def recurrence_step_kernel(size: str, sequences: int, peaks) -> dict:
    *_, heads, key, value, _ = SIZES[size]
    o, rank = hybrid.Ops("bfloat16"), 16
    width = 2 * heads * (key + value) + rank
    one = torch.ones(sequences, dtype=torch.int32, device="cuda")
    first = torch.arange(sequences, dtype=torch.int32, device="cuda")
    decay, bias, norm = normal(heads * key, rank), normal(heads * key), normal(value)

    def make(i):
        state, projected, out = normal(sequences, heads, key, value, kind=torch.float32), o.rows(sequences, width), o.rows(sequences, heads * value)
        projected.normal_()
        return lambda: o.call("singe_gated_linear_step_bf16", _stream(), out, out.stride(0), projected, projected.stride(0), decay, bias,
                              norm, state, first, one, one, sequences, sequences, heads, key, value, rank, 16.0, key ** -0.5, 1e-6, 8)

    moved = sequences * (8 * heads * key * value + 2 * width + 2 * heads * value)
    call, _ = rotating(make, moved)
    return {"shape": f"{sequences} x {heads} heads, state {key} x {value}", **_memory(graph_seconds(call), moved, peaks)}


def recurrence_prompt_kernel(size: str, lengths, peaks) -> dict:
    from singe_b200 import kernel_sys as ks

    *_, heads, key, value, _ = SIZES[size]
    o, rank, total = hybrid.Ops("bfloat16"), 16, sum(lengths)
    width = 2 * heads * (key + value) + rank
    projected, out = o.rows(total, width), o.rows(total, heads * value)
    projected.normal_()
    decay, bias, norm = normal(heads * key, rank, scale=0.25), normal(heads * key) + 2.0, normal(value)
    state = torch.zeros((len(lengths), heads, key, value), device="cuda")
    context = torch.zeros(len(lengths), dtype=torch.int32, device="cuda")
    firsts = np.cumsum([0] + lengths)[:-1]
    starts = [np.arange(f, f + n, 16) for f, n in zip(firsts, lengths)]
    plan = np.asarray(hybrid.plan_segments([len(s) for s in starts], heads, torch.cuda.get_device_properties(0).multi_processor_count))
    i32 = lambda a: torch.tensor(np.ascontiguousarray(a), dtype=torch.int32, device="cuda")
    tokens = np.concatenate([np.minimum(f + n - s, 16) for f, n, s in zip(firsts, lengths, starts)])
    rows, tokens, segments, last = i32(np.concatenate(starts)), i32(tokens), i32(plan[:, :4]), i32(plan[:, 4])
    scratch = torch.empty(int(ks.lib().singe_gated_linear_prompt_scratch(heads, key, value, rows.numel(), len(plan))), dtype=torch.uint8, device="cuda")
    call = lambda: o.call("singe_gated_linear_prompt_bf16", _stream(), out, out.stride(0), projected, projected.stride(0), decay, bias, norm,
                          state, context, total, heads, key, value, rank, 16.0, key ** -0.5, 1e-6, rows, tokens, rows.numel(), segments, last,
                          len(plan), int((plan[:, 4] == 0).any()), scratch)
    moved = 2 * total * (width + heads * value)
    return {"shape": f"{len(lengths)} x {lengths[0]} tokens, {heads} heads, state {key} x {value}, {len(plan)} segments",
            **_memory(graph_seconds(call, 4), moved, peaks)}


def glue_kernels(size: str, rows: int, peaks) -> dict:
    width, heads, dim, q_rank, kv_rank, _, ffn, *_ = SIZES[size]
    o = hybrid.Ops("bfloat16")
    out = {}

    def layer_norm(i):
        residual, delta, normed, weight = torch.randn((rows, width), device="cuda"), normal(rows, width), o.rows(rows, width), normal(width)
        return lambda: o.add_layer_norm(_stream(), residual, delta, normed, weight, 1e-6)

    def rms_norm(i):
        hidden, delta, normed, weight = normal(rows, width), normal(rows, width), normal(rows, width), normal(width)
        return lambda: o.call("singe_add_rms_norm_bf16", _stream(), hidden, delta, normed, weight, rows, width, 1e-6)

    def latent_norm(i):
        projected, q_out, cache = o.rows(rows, q_rank + kv_rank + heads), o.rows(rows, q_rank), normal(-(-rows // 16), 16, kv_rank)
        projected.normal_()
        index = torch.arange(rows, device="cuda")
        pages, slots, qw, kw = index // 16, index % 16, normal(q_rank), normal(kv_rank)
        return lambda: o.call("singe_latent_norm_cache_write_bf16", _stream(), q_out, q_out.stride(0), cache, kv_rank, projected,
                              projected.stride(0), qw, q_rank, kw, kv_rank, pages, slots, rows, cache.shape[0], 16, 1e-6, None)

    def rotary(i):
        kv = heads // 4
        qkv, query = normal(rows, (heads + 2 * kv) * dim), normal(rows, heads, dim)
        keys, values = normal(-(-rows // 16), 16, kv, dim), normal(-(-rows // 16), 16, kv, dim)
        index = torch.arange(rows, device="cuda")
        pages, slots, cos, sin = index // 16, index % 16, normal(rows, dim // 2), normal(rows, dim // 2)
        return lambda: o.call("singe_rotary_cache_write_bf16", _stream(), query, qkv, qkv.stride(0), cos, sin, index, keys, values,
                              pages, slots, 8, rows, heads, kv, dim, keys.shape[0], 16, rows, None)

    kv = heads // 4
    for name, make, moved in (("add_layer_norm (f32 residual)", layer_norm, rows * width * 12),
                              ("llama add_rms_norm (bf16 residual)", rms_norm, rows * width * 8),
                              ("latent norms + cache write", latent_norm, 4 * rows * (q_rank + kv_rank)),
                              ("llama rotary + cache write", rotary, 4 * rows * (heads + 2 * kv) * dim)):
        call, _ = rotating(make, moved)
        out[name] = _memory(graph_seconds(call), moved, peaks)
    return out


def linear_kernels(size: str, rows: int, peaks) -> dict:
    """The linears of a layer; a decode batch streams its weights, a prompt is bound by the tensor core."""
    width, heads, dim, q_rank, kv_rank, _, ffn, gla_heads, key, value, _ = SIZES[size]
    o = hybrid.Ops("bfloat16")
    shapes = {"down projections": (q_rank + kv_rank + heads, width, 0), "query up": (heads * dim, q_rank, 0),
              "output": (width, heads * dim, 0), "up + squared relu": (ffn, width, 2), "down": (width, ffn, 0),
              "recurrence in": (2 * gla_heads * (key + value) + 16, width, 0), "keys and values": (2 * heads * dim, kv_rank, 0),
              "llama qkv": ((heads + heads // 2) * dim, width, 0), "llama gate/up + swiglu": (2 * ffn, width, 1)}
    out = {}
    for name, (n, k, activation) in shapes.items():
        x = normal(rows, k)
        y = o.rows(rows, n // 2 if activation == 1 else n)

        def make(i):
            w = normal(n, k, scale=k ** -0.5)
            return lambda: o.linear(_stream(), y, x, w, activation)

        if rows <= 128:
            call, _ = rotating(make, n * k * 2)
            out[name] = {"shape": f"{rows} x {n} x {k}", **_memory(graph_seconds(call), 2 * (n * k + rows * (n + k)), peaks)}
        else:
            out[name] = {"shape": f"{rows} x {n} x {k}", **_compute(graph_seconds(make(0), 4), 2.0 * rows * n * k, peaks)}
    if rows <= 128:
        for name, n, k in (("absorb per head", kv_rank, dim), ("values per head", dim, kv_rank)):
            x, y = normal(rows, heads * k), o.rows(rows, heads * n)

            def make(i):
                w = normal(heads, n, k)
                return lambda: o.head_linear(_stream(), y, x, w, heads)

            moved = 2 * heads * (n * k + rows * (n + k))
            call, _ = rotating(make, moved)
            out[name] = {"shape": f"{heads} x ({rows} x {n} x {k})", **_memory(graph_seconds(call), moved, peaks)}
    return out


def kernel_figures(size: str, peaks) -> dict:
    torch.manual_seed(0)
    out = {"decode attention": {f"{s} x {c}": {"kavalorn": latent_decode_kernel(size, s, c, peaks), "llama": paged_decode_kernel(size, s, c, peaks)}
                                for s, c in ((64, 2048), (8, 8192), (64, 4096))},
           "prompt attention": {f"{len(l)} x {l[0]}": prompt_attention_kernels(size, l, peaks) for l in ([8192], [2048] * 4)},
           "recurrence, one token": {str(s): recurrence_step_kernel(size, s, peaks) for s in (64, 8)},
           "recurrence, prompt": {f"{len(l)} x {l[0]}": recurrence_prompt_kernel(size, l, peaks) for l in ([8192], [2048] * 4, [512] * 16)},
           "glue, 64 rows": glue_kernels(size, 64, peaks), "glue, 8192 rows": glue_kernels(size, 8192, peaks),
           "linears, 64 rows": linear_kernels(size, 64, peaks), "linears, 8192 rows": linear_kernels(size, 8192, peaks)}
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
