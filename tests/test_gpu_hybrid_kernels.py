"""Each mechanism of the layer-list decoder alone, against the plain float64 restatement in ``oracle.hybrid_ref``."""
import numpy as np
import pytest
import torch

from oracle import hybrid_ref
from singe_b200 import kernel_sys as ks
from singe_b200.hybrid import Ops, plan_segments
from tests.gpu_util import dev, dev_u32, host
from tests.hybrid_util import bf16

pytestmark = pytest.mark.gpu


def stream():
    return int(torch.cuda.current_stream().cuda_stream)


def i32(values):
    return torch.tensor(np.asarray(values), dtype=torch.int32, device="cuda")


def i64(values):
    return torch.tensor(np.asarray(values), dtype=torch.int64, device="cuda")


def relative(got, expect):
    """Root mean square of the difference over that of the expectation, worst row."""
    got, expect = np.asarray(got, dtype=np.float64), np.asarray(expect, dtype=np.float64)
    got, expect = got.reshape(-1, got.shape[-1]), expect.reshape(-1, expect.shape[-1])
    scale = np.sqrt((expect ** 2).mean(1)) + 1e-12
    return float((np.sqrt(((got - expect) ** 2).mean(1)) / scale).max())


def draw(rng, *shape, scale=1.0, exact16=True):
    values = (rng.standard_normal(shape) * scale).astype(np.float32)
    return bf16(values) if exact16 else values


LIMIT = {"bfloat16": 6e-3, "float32": 2e-6}


# ---- norms ----

@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("rows,width", [(1, 1), (3, 7), (5, 100), (4, 4096), (2, 1028), (2, 16384), (3, 3001)])
def test_layer_norm_with_residual_add(dtype, rows, width):
    rng = np.random.default_rng(rows * width)
    ops = Ops(dtype)
    residual = draw(rng, rows, width, exact16=False) + 300.0   # a mean far from zero: squares must be of deviations
    delta, weight = draw(rng, rows, width), draw(rng, width)
    d_residual, d_delta = dev(residual), ops.weight(delta)
    normed = ops.rows(rows, width)
    ops.add_layer_norm(stream(), d_residual, d_delta, normed, ops.weight(weight), 1e-3)
    total = residual + delta
    assert np.array_equal(host(d_residual), total.astype(np.float32))
    expect = hybrid_ref.layer_norm(total.astype(np.float64), weight, 1e-3)
    if width > 1:
        assert (np.abs(host(normed) - expect) / (1.0 + np.abs(expect))).max() <= (1e-2 if dtype == "bfloat16" else 2e-3)
        assert relative(host(normed), expect) < {"bfloat16": 6e-3, "float32": 3e-4}[dtype]
    else:
        assert np.abs(host(normed)).max() == 0.0
    small = dev(residual - 300.0)
    ops.add_layer_norm(stream(), small, None, normed, ops.weight(weight), 1e-3)
    if width > 1:
        assert relative(host(normed), hybrid_ref.layer_norm((residual - 300.0).astype(np.float64), weight, 1e-3)) < LIMIT[dtype]


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_eps_sits_inside_the_root(dtype):
    ops = Ops(dtype)
    x = np.zeros((1, 64), dtype=np.float32)
    x[0, 0] = 1e-2
    normed = ops.rows(1, 64)
    ops.add_layer_norm(stream(), dev(x), None, normed, ops.weight(np.ones(64, dtype=np.float32)), 0.5)
    assert relative(host(normed), hybrid_ref.layer_norm(x.astype(np.float64), np.ones(64), 0.5)) < LIMIT[dtype]


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("width", [13, 96, 4096])
def test_embedding_with_its_norm(dtype, width):
    rng = np.random.default_rng(width)
    ops = Ops(dtype)
    table, weight, ids = draw(rng, 37, width), draw(rng, width), np.array([0, 36, 5, 5, -1, 99])
    residual = torch.empty((6, width), dtype=torch.float32, device="cuda")
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    ops.call(f"singe_embedding_layer_norm_{ops.suffix}", stream(), residual, dev(table).to(ops.dtype), i64(ids),
             dev(weight).to(ops.dtype), 6, width, 37, 1e-6, status)
    expect = hybrid_ref.layer_norm(table[[0, 36, 5, 5, 36]].astype(np.float64), weight, 1e-6)
    assert relative(host(residual)[:5], expect) < 2e-6   # f32 whatever the weights' type
    assert int(status.item()) == 1


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("q_rank,kv_rank,cache_width", [(24, 40, 64), (7, 5, 8), (72, 104, 128), (1536, 512, 512)])
def test_latent_norms_and_cache_write(dtype, q_rank, kv_rank, cache_width):
    rng = np.random.default_rng(q_rank)
    ops = Ops(dtype)
    tokens, pages, page_size = 5, 4, 3
    x = draw(rng, tokens, q_rank + kv_rank + 3)
    q_weight, kv_weight = draw(rng, q_rank), draw(rng, kv_rank)
    write_pages, write_slots = [3, 0, 2, 2, 9], [1, 2, 0, 1, 0]   # the last one is outside
    cache = torch.full((pages, page_size, 1, cache_width), 7.0, dtype=ops.dtype, device="cuda")
    q_out, projected = ops.rows(tokens, q_rank), ops.weight(x)
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    ops.call(f"singe_latent_norm_cache_write_{ops.suffix}", stream(), q_out, q_out.stride(0), cache, cache_width, projected,
             projected.stride(0), ops.weight(q_weight), q_rank, ops.weight(kv_weight), kv_rank, i64(write_pages),
             i64(write_slots), tokens, pages, page_size, 1e-4, status)
    assert relative(host(q_out), hybrid_ref.rms_norm(x[:, :q_rank].astype(np.float64), q_weight, 1e-4)) < LIMIT[dtype]
    expect = hybrid_ref.rms_norm(x[:, q_rank:q_rank + kv_rank].astype(np.float64), kv_weight, 1e-4)
    stored = host(cache)[:, :, 0]
    for t in range(4):
        row = stored[write_pages[t], write_slots[t]]
        assert relative(row[None, :kv_rank], expect[t][None]) < LIMIT[dtype] and (row[kv_rank:] == 0).all()
    assert int(status.item()) == 1 and (stored[1] == 7.0).all()


# ---- linears ----

@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("m,n,k", [(1, 1, 1), (3, 5, 7), (64, 184, 96), (130, 72, 24), (300, 513, 100), (17, 3584, 640)])
def test_linear_with_squared_relu(dtype, m, n, k):
    rng = np.random.default_rng(m + n + k)
    ops = Ops(dtype)
    x, w = draw(rng, m, k), draw(rng, n, k, scale=k ** -0.5)
    for activation in (0, 2):
        out = ops.rows(m, n)
        ops.linear(stream(), out, ops.weight(x), ops.weight(w), activation)
        expect = x.astype(np.float64) @ w.T.astype(np.float64)
        if activation:
            expect = np.maximum(expect, 0.0) ** 2
        worst = np.abs(host(out) - expect) / (np.abs(expect) + 1.0)
        assert worst.max() < {"bfloat16": 8e-3, "float32": 5e-6}[dtype]
    logits = torch.empty((m, n), dtype=torch.float32, device="cuda")
    ops.linear_f32_out(stream(), logits, ops.weight(x), ops.weight(w))
    assert np.abs(host(logits) - x.astype(np.float64) @ w.T).max() < 1e-4


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("rows,heads,columns,reduction", [(1, 1, 8, 8), (5, 3, 27, 16), (64, 5, 64, 72), (130, 2, 512, 128),
                                                          (257, 7, 128, 320)])
@pytest.mark.parametrize("gated", [False, True])
def test_one_product_per_head(dtype, rows, heads, columns, reduction, gated):
    rng = np.random.default_rng(rows * heads + columns)
    ops = Ops(dtype)
    x, w = draw(rng, rows, heads * reduction), draw(rng, heads, columns, reduction, scale=reduction ** -0.5)
    gate = draw(rng, rows, heads, scale=3.0)
    out = ops.rows(rows, heads * columns)
    gates = ops.weight(np.concatenate([gate, gate], 1))[:, heads:] if gated else None
    ops.head_linear(stream(), out, ops.weight(x), dev(w).to(ops.dtype), heads, gates)
    expect = np.einsum("thk,hnk->thn", x.reshape(rows, heads, reduction).astype(np.float64), w.astype(np.float64))
    if gated:
        expect = expect * hybrid_ref.sigmoid(gate.astype(np.float64))[:, :, None]
    got = host(out).reshape(rows, heads, columns)
    assert (np.abs(got - expect) / (np.abs(expect) + 1.0)).max() < {"bfloat16": 8e-3, "float32": 5e-6}[dtype]


# ---- attention over latents ----

def edge_queries(rng, keys, positions, window, heads, sharp=30.0):
    """Queries that single out one key each: the last one the window still holds, the first one it no longer does, the
    token itself, and one far back, by turns -- one key too many or too few changes the whole row."""
    dim = keys.shape[-1]
    unit = keys / np.linalg.norm(keys, axis=-1, keepdims=True)
    query = np.zeros((len(positions), heads, dim), dtype=np.float32)
    for row, position in enumerate(positions):
        for h in range(heads):
            target = (position - window + 1, position - window, position, position // 3)[(row + h) % 4]
            target = min(max(target, 0), position)
            query[row, h] = sharp * unit[target, h % unit.shape[1]]
    return bf16(query + 0.05 * rng.standard_normal(query.shape))


@pytest.mark.parametrize("heads,latent,page_size,window,splits", [
    (1, 64, 16, 1, 1), (5, 64, 16, 2, 1), (9, 128, 16, 150, 3), (16, 192, 4, 65, 2), (20, 256, 7, 64, 1),
    (34, 512, 16, 300, 4), (32, 320, 16, 100000, 7), (3, 448, 1, 33, 5), (40, 64, 16, 0, 2),
    (32, 512, 64, 200, 2), (8, 256, 128, 129, 1), (33, 320, 64, 64, 3), (4, 64, 8, 77, 2), (16, 448, 32, 1, 1)])
def test_decode_attention_at_window_and_page_edges(heads, latent, page_size, window, splits):
    rng = np.random.default_rng(heads * latent + window)
    capacity = 500
    lens = np.array([1, 2, 500, 0, page_size, page_size + 1, max(window, 1), window + 1, window + 2, 63, 64, 65, 129, 317])
    lens = np.minimum(lens, capacity)
    sequences = len(lens)
    stride = -(-capacity // page_size)
    pages = sequences * stride + 3
    table = rng.permutation(pages)[: sequences * stride].reshape(sequences, stride).astype(np.uint32)
    cache = draw(rng, pages, page_size, latent)
    order = rng.permutation(sequences)     # query i reads sequence order[i]
    scale = 1.0 / np.sqrt(latent)
    queries, expect = [], []
    for b in order:
        rows = np.array([cache[table[b, j // page_size], j % page_size] for j in range(lens[b])]).reshape(-1, latent)
        if lens[b] == 0:
            queries.append(draw(rng, heads, latent))
            expect.append(np.zeros((heads, latent)))
            continue
        seen = window if window > 0 else capacity
        q = edge_queries(rng, rows[:, None], [lens[b] - 1], seen, heads)[0]
        queries.append(q)
        first = max(0, lens[b] - seen)
        score = (q.astype(np.float64) @ rows[first:].T.astype(np.float64)) * scale
        weight = np.exp(score - score.max(1, keepdims=True))
        expect.append(weight / weight.sum(1, keepdims=True) @ rows[first:].astype(np.float64))
    query = dev(np.stack(queries)).to(torch.bfloat16)
    out = torch.full(query.shape, float("nan"), dtype=torch.bfloat16, device="cuda")
    attn = torch.full((sequences, splits, heads, latent), float("nan"), device="cuda")
    lse = torch.full((sequences, splits, heads), float("nan"), device="cuda")
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    Ops("bfloat16").call("singe_latent_decode_bf16", stream(), out, attn, lse, query, dev(cache).to(torch.bfloat16),
                         i32(order), i32(lens[order]), dev_u32(table), sequences, heads, latent, page_size, pages, sequences,
                         stride, window, splits, scale, status)
    got = host(out)
    assert np.isfinite(got).all() and int(status.item()) == 0
    error = np.abs(got - np.stack(expect)) / (1.0 + np.abs(np.stack(expect)))
    assert error.max() < 1e-2, f"query, head, column {np.unravel_index(error.argmax(), error.shape)}: {error.max()}"


def test_decode_attention_reports_bad_pages():
    cache = torch.zeros((2, 16, 64), dtype=torch.bfloat16, device="cuda")
    query = torch.ones((2, 4, 64), dtype=torch.bfloat16, device="cuda")
    out = torch.empty_like(query)
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    call = lambda sequence, table: Ops("bfloat16").call(
        "singe_latent_decode_bf16", stream(), out, None, None, query, cache, i32(sequence), i32([20, 20]), i32(table), 2, 4, 64,
        16, 2, 2, 2, 0, 1, 1.0, status)
    call([0, 1], [[0, 1], [1, 2]])
    assert int(status.item()) == 1
    status.zero_()
    call([0, 2], [[0, 1], [1, 0]])
    assert int(status.item()) == 1


@pytest.mark.parametrize("heads,size,window", [(2, 64, 1), (3, 64, 2), (1, 128, 127), (2, 64, 128), (2, 128, 129), (1, 64, 250),
                                               (2, 128, 300), (3, 64, 100000)])
def test_prompt_attention_at_window_edges(heads, size, window):
    rng = np.random.default_rng(size + window)
    contexts, fresh = [0, 0, 37, 200, 511, 0], [1, 300, 130, 257, 9, 128]
    kept = [min(context, window - 1) for context in contexts]     # the keys before the portion that it still sees
    lens_kv = np.array([k + n for k, n in zip(kept, fresh)])
    offsets_q = np.cumsum([3] + fresh)[:-1]                       # the packed rows need not start at zero
    offsets_kv = np.cumsum([5] + list(lens_kv))[:-1]
    total_q, total_kv = offsets_q[-1] + fresh[-1] + 2, offsets_kv[-1] + lens_kv[-1] + 1
    rows = draw(rng, total_kv, 2, heads, size)
    query, gate = np.zeros((total_q, heads, size), dtype=np.float32), draw(rng, total_q, heads + 2)
    scale = 1.0 / np.sqrt(size)
    expect = {}
    for b, n in enumerate(fresh):
        keys, values = (rows[offsets_kv[b]: offsets_kv[b] + lens_kv[b], i] for i in (0, 1))
        positions = np.arange(kept[b], lens_kv[b])
        q = edge_queries(rng, keys, positions, window, heads)
        query[offsets_q[b]: offsets_q[b] + n] = q
        padded = np.concatenate([np.zeros((kept[b], heads, size)), q])
        full = hybrid_ref.windowed_attention(padded, keys.astype(np.float64), values.astype(np.float64), scale, window)
        gates = hybrid_ref.sigmoid(gate[offsets_q[b]: offsets_q[b] + n, 2:].astype(np.float64))
        expect[b] = full[kept[b]:] * gates[:, :, None]
    ops = Ops("bfloat16")
    d_rows, d_gate = dev(rows).to(torch.bfloat16), dev(gate).to(torch.bfloat16)
    out = torch.zeros((total_q, heads, size), dtype=torch.bfloat16, device="cuda")
    lse = torch.zeros((total_q, heads), dtype=torch.float32, device="cuda")
    ops.call("singe_windowed_prefill_attention_bf16", stream(), out, lse, dev(query).to(torch.bfloat16), d_rows,
             d_rows.data_ptr() + heads * size * 2, 2 * heads * size, i32(fresh), i32(lens_kv), i32(offsets_q),
             i32(offsets_kv), d_gate.data_ptr() + 4, gate.shape[1], len(fresh), total_q, total_kv, heads, heads, size, window, scale)
    got = host(out)
    for b, n in enumerate(fresh):
        assert np.abs(got[offsets_q[b]: offsets_q[b] + n] - expect[b]).max() < 3e-2, f"sequence {b}"
    assert ks.lib().singe_take_device_error(None) == 0


@pytest.mark.parametrize("window", [90, 400])
def test_prompt_attention_with_scores_that_leave_the_single_pass_range(window):
    """Scores that jump by hundreds from one key tile to the next, up and down, also in a row's first visible tile."""
    rng = np.random.default_rng(window)
    tokens, heads, size = 640, 2, 64
    rows, query = draw(rng, tokens, 2, heads, size), draw(rng, tokens, heads, size)
    rows[:, 0] *= np.where((np.arange(tokens) // 100) % 2 == 0, 40.0, 0.1).astype(np.float32)[:, None, None]
    rows, query = bf16(rows), bf16(query * 8.0)
    expect = hybrid_ref.windowed_attention(query.astype(np.float64), rows[:, 0].astype(np.float64),
                                           rows[:, 1].astype(np.float64), 1.0, window)
    ops = Ops("bfloat16")
    d_rows = dev(rows).to(torch.bfloat16)
    out = torch.zeros((tokens, heads, size), dtype=torch.bfloat16, device="cuda")
    lse = torch.zeros((tokens, heads), dtype=torch.float32, device="cuda")
    ops.call("singe_windowed_prefill_attention_bf16", stream(), out, lse, dev(query).to(torch.bfloat16), d_rows,
             d_rows.data_ptr() + heads * size * 2, 2 * heads * size, i32([tokens]), i32([tokens]), i32([0]), i32([0]), None, 0,
             1, tokens, tokens, heads, heads, size, window, 1.0)
    assert np.abs(host(out) - expect).max() < 3e-2


# ---- the recurrence ----

def recurrence_case(rng, counts, heads, dim, vdim, rank, bias, spread):
    """Projected rows of sequences with ``counts`` new tokens (an idle row for none), weights, and the f64 parts."""
    rows = int(sum(max(n, 1) for n in counts))
    x = draw(rng, rows, 2 * heads * (dim + vdim) + rank)
    a2, b = draw(rng, heads * dim, rank, scale=spread), bf16(bias + draw(rng, heads * dim, scale=spread))
    return x, a2, b, draw(rng, vdim)


def recurrence_expect(x, a2, b, norm, first, n, state, heads, dim, vdim, rank, tau, eps):
    part = x[first: first + n].astype(np.float64)
    keys, values = heads * dim, heads * vdim
    query = part[:, :keys].reshape(n, heads, dim) / np.sqrt(dim)
    key = part[:, keys:2 * keys].reshape(n, heads, dim)
    value = part[:, 2 * keys:2 * keys + values].reshape(n, heads, vdim)
    gate = part[:, 2 * keys + values:2 * keys + 2 * values].reshape(n, heads, vdim)
    z = (part[:, 2 * keys + 2 * values:] @ a2.T + b).reshape(n, heads, dim)
    out, state = hybrid_ref.gated_recurrence(query, key, value, hybrid_ref.sigmoid(z) ** (1.0 / tau), state)
    return hybrid_ref.rms_norm(out, norm, eps) * gate * hybrid_ref.sigmoid(gate), state


CASES = [  # heads, dim, vdim, rank, tau, bias, spread
    (3, 56, 80, 20, 12.0, 2.0, 1.0),
    (3, 24, 40, 5, 4.0, 2.0, 1.0),
    (1, 8, 8, 1, 1.0, 0.0, 2.0),
    (2, 128, 256, 24, 10.0, 2.0, 0.5),
    (1, 256, 128, 8, 8.0, 1.0, 0.5),
    (4, 64, 128, 16, 1.0, -6.0, 3.0),     # decays too strong to factor
    (2, 16, 272, 3, 2.0, -3.0, 6.0),      # some blocks are, some are not
]


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("heads,dim,vdim,rank,tau,bias,spread", CASES + [(2, 10, 13, 7, 2.5, 1.0, 1.0), (1, 33, 300, 4, 3.0, 1.0, 1.0)])
def test_recurrence_token_by_token(dtype, heads, dim, vdim, rank, tau, bias, spread):
    rng = np.random.default_rng(dim * vdim)
    counts, contexts = [1, 0, 3, 7, 1], [0, 5, 0, 4, 9]
    x, a2, b, norm = recurrence_case(rng, counts, heads, dim, vdim, rank, bias, spread)
    before = draw(rng, 5, heads, dim, vdim, exact16=False)
    ops = Ops(dtype)
    first = np.cumsum([0] + [max(n, 1) for n in counts])[:-1]
    state, projected, out = dev(before), ops.weight(x), ops.rows(len(x), heads * vdim)
    out.fill_(float("nan"))
    ops.call(f"singe_gated_linear_step_{ops.suffix}", stream(), out, out.stride(0), projected, projected.stride(0),
             dev(a2).to(ops.dtype), dev(b).to(ops.dtype), dev(norm).to(ops.dtype), state, i32(first), i32(counts),
             i32(contexts), len(x), 5, heads, dim, vdim, rank, tau, dim ** -0.5, 1e-5, 5)
    got = host(out).reshape(-1, heads, vdim)
    after = host(state)
    for s, n in enumerate(counts):
        if n == 0:
            assert (got[first[s]] == 0).all() and np.array_equal(after[s], before[s])
        elif n > 5:
            assert np.isnan(got[first[s]: first[s] + n]).all() and np.array_equal(after[s], before[s])
        else:
            start = before[s].astype(np.float64) * (contexts[s] > 0)
            expect, end = recurrence_expect(x, a2, b, norm, first[s], n, start, heads, dim, vdim, rank, tau, 1e-5)
            assert relative(got[first[s]: first[s] + n], expect) < {"bfloat16": 6e-3, "float32": 5e-5}[dtype]
            assert relative(after[s], end) < 1e-5


@pytest.mark.parametrize("heads,dim,vdim,rank,tau,bias,spread", CASES)
def test_recurrence_block_by_block(heads, dim, vdim, rank, tau, bias, spread):
    rng = np.random.default_rng(dim + vdim + heads)
    counts, contexts = [16, 9, 1, 333, 15, 17, 600], [0, 3, 7, 0, 0, 20, 5]
    sequences = len(counts)
    x, a2, b, norm = recurrence_case(rng, counts, heads, dim, vdim, rank, bias, spread)
    before = draw(rng, sequences, heads, dim, vdim, exact16=False)
    first = np.cumsum([0] + counts)[:-1]
    served = [s for s, n in enumerate(counts) if n > 8]
    starts = [np.arange(first[s], first[s] + counts[s], 16) for s in served]
    tokens = np.concatenate([np.minimum(first[s] + counts[s] - start, 16) for s, start in zip(served, starts)])
    plan = np.asarray(plan_segments([len(start) for start in starts], heads, 148))
    assert (plan[:, 4] == 0).any()
    segments = np.stack([np.asarray(served)[plan[:, 0]], plan[:, 1], plan[:, 2], plan[:, 3]], 1)
    ops = Ops("bfloat16")
    state, projected, out = dev(before), ops.weight(x), ops.rows(len(x), heads * vdim)
    out.fill_(float("nan"))
    size = int(ks.lib().singe_gated_linear_prompt_scratch(heads, dim, vdim, len(tokens), len(plan)))
    assert size > 0
    ops.call("singe_gated_linear_prompt_bf16", stream(), out, out.stride(0), projected, projected.stride(0),
             dev(a2).to(ops.dtype), dev(b).to(ops.dtype), dev(norm).to(ops.dtype), state, i32(contexts), len(x), heads, dim, vdim, rank,
             tau, dim ** -0.5, 1e-5, i32(np.concatenate(starts)), i32(tokens), len(tokens), i32(segments), i32(plan[:, 4]),
             len(plan), 1, torch.empty(size, dtype=torch.uint8, device="cuda"))
    got, after = host(out).reshape(-1, heads, vdim), host(state)
    for s, n in enumerate(counts):
        if s not in served:
            assert np.array_equal(after[s], before[s]) and np.isnan(got[first[s]: first[s] + n]).all()
            continue
        start = before[s].astype(np.float64) * (contexts[s] > 0)
        expect, end = recurrence_expect(x, a2, b, norm, first[s], n, start, heads, dim, vdim, rank, tau, 1e-5)
        assert relative(got[first[s]: first[s] + n], expect) < 6e-3, f"sequence {s}"
        assert relative(after[s], end) < 1e-4, f"state of sequence {s}"   # far below what one bf16 rounding would leave


def test_argmax_over_f32_logits_breaks_ties_low():
    logits = torch.zeros((3, 1000), device="cuda")
    logits[0, 7] = logits[0, 900] = 1.0
    logits[1, 3] = float("nan")
    logits[1, 999] = 1e-7
    value = torch.empty(3, device="cuda")
    index = torch.empty(3, dtype=torch.int64, device="cuda")
    Ops("float32").call("singe_argmax_f32", stream(), value, index, logits, 1000, 3, 1000, 10)
    assert index.tolist() == [17, 1009, 10]
