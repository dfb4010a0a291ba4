"""Each mechanism of the Vatolorn decoder alone, against the plain float64 restatement in ``oracle.vatolorn_ref``."""
import numpy as np
import pytest
import torch

from oracle import vatolorn_ref as ref
from singe_b200 import kernel_sys as ks
from singe_b200.layer_ops import Ops, round_up
from singe_b200.parallel_mixer import NO_WINDOW, Rotation, YarnScaling
from tests.gpu_util import dev, host
from tests.hybrid_util import bf16
from tests.test_gpu_hybrid_kernels import draw, i32, i64, relative, stream

pytestmark = pytest.mark.gpu

LIMIT = {"bfloat16": 6e-3, "float32": 5e-6}


# ---- several residual streams ----

@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("parts", [1, 2])
@pytest.mark.parametrize("rows,streams,width", [(3, 1, 96), (5, 2, 100), (2, 3, 7), (4, 4, 4096), (3, 5, 1028), (2, 8, 256), (2, 16, 33)])
def test_streams_take_a_sublayer_in(dtype, parts, rows, streams, width):
    rng = np.random.default_rng(rows * streams * width + parts)
    ops, eps = Ops(dtype), 1e-4
    before = draw(rng, rows, streams, width, exact16=False)
    sides = [draw(rng, rows, width, scale=3.0) for _ in range(parts)]
    gains = [draw(rng, width) for _ in range(parts)]
    blend_in, blend_out, blend_mix = [draw(rng, *shape) for shape in ((streams,), (streams,), (streams, streams))]
    weight = draw(rng, width)
    second_at = round_up(width, 8)
    delta = ops.rows(rows, width if parts == 1 else second_at + width)
    for side, values in enumerate(sides):
        delta[:, side * second_at: side * second_at + width] = dev(values).to(ops.dtype)
    d_gains = [ops.weight(gain) for gain in gains] if parts == 2 else [None, None]
    d_streams, normed = dev(before), ops.rows(rows, width)
    scalars = [ops.scalars(values) for values in (blend_mix, blend_out, blend_in)]
    ops.call(f"singe_stream_step_norm_{ops.suffix}", stream(), d_streams, delta, delta.stride(0), parts, second_at, *d_gains, 0.5,
             *scalars, 1, normed, normed.stride(0), ops.weight(weight), 0.75, rows, streams, width, eps)
    y = sides[0] if parts == 1 else 0.5 * sum(ref.rms_norm(side.astype(np.float64), gain, eps) for side, gain in zip(sides, gains))
    after = ref.stream_step(before.transpose(1, 0, 2).astype(np.float64), lambda u: y, {"in": blend_in, "out": blend_out, "mix": blend_mix})
    assert relative(host(d_streams), after.transpose(1, 0, 2)) < 5e-6
    expect = ref.rms_norm(np.einsum("s,stw->tw", blend_in, after), weight, eps) * 0.75
    assert relative(host(normed), expect) < LIMIT[dtype]


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("streams,width", [(1, 64), (3, 99), (4, 512), (6, 40)])
def test_streams_start_as_the_embedding(dtype, streams, width):
    rng = np.random.default_rng(streams * width)
    ops, table, blend, weight = Ops(dtype), draw(rng, 11, width), draw(rng, streams), draw(rng, width)
    ids = [3, 10, 0, -1]
    d_streams = torch.full((4, streams, width), float("nan"), device="cuda")
    normed, status = ops.rows(4, width), torch.zeros(1, dtype=torch.int32, device="cuda")
    run = lambda ids: ops.call(f"singe_stream_embedding_norm_{ops.suffix}", stream(), d_streams, dev(table).to(ops.dtype), i64(ids),
                               ops.scalars(blend), normed, normed.stride(0), ops.weight(weight), 4, streams, width, 11, 1e-5, status)
    run(ids)
    assert np.array_equal(host(d_streams), np.repeat(table[ids][:, None], streams, 1))
    expect = ref.rms_norm(blend.astype(np.float64).sum() * table[ids].astype(np.float64), weight, 1e-5)
    assert relative(host(normed), expect) < LIMIT[dtype] and int(status.item()) == 0
    run([0, 11, 1, 2])
    assert int(status.item()) == ks.STATUS_INDEX_OUT_OF_BOUNDS


# ---- short convolutions ----

def portions(total, sizes):
    at = 0
    while at < total:
        for size in sizes:
            if at < total:
                yield at, min(size, total - at)
                at += size


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("taps,heads,dim,rest", [(1, 1, 8, 8), (2, 2, 10, 13), (4, 3, 24, 40), (5, 2, 64, 128), (9, 1, 3, 5)])
@pytest.mark.parametrize("sizes", [(64,), (1,), (2, 1, 7), (3, 1, 1, 16)])
def test_convolution_with_silu_and_unit_lengths_over_portions(dtype, taps, heads, dim, rest, sizes):
    """Two sequences in rows 2 and 0 of three, the state carried from portion to portion; row 1 idles."""
    rng = np.random.default_rng(taps * dim)
    ops, total = Ops(dtype), 37
    second_at = round_up(heads * dim, 8)
    span = second_at + round_up(heads * dim, 8) + rest
    projected, weight = draw(rng, 2, total, span), draw(rng, taps, span, scale=taps ** -0.5)
    state = torch.full((3, taps - 1, span), float("nan"), dtype=ops.dtype, device="cuda")
    d_taps = dev(weight).to(ops.dtype)
    mixed_all, inverse_all = np.zeros((2, total, span)), np.zeros((2, total, 2 * heads))
    for at, n in portions(total, sizes):
        fresh, context, first = [n, 0, n], [at, 3, at], [0, n, n + 1]
        rows = ops.rows(2 * n + 1, span)
        rows.fill_(float("nan"))
        rows[:n], rows[n + 1:] = dev(projected[0, at: at + n]).to(ops.dtype), dev(projected[1, at: at + n]).to(ops.dtype)
        mixed = ops.rows(2 * n + 1, span)
        mixed.fill_(float("nan"))
        inverse = torch.empty((2 * n + 1, 2 * heads), device="cuda")
        d_first, d_fresh = i32(first), i32(fresh)
        ops.call(f"singe_conv_recurrence_inputs_{ops.suffix}", stream(), mixed, mixed.stride(0), inverse, rows, rows.stride(0), d_taps,
                 state, i32([0] * n + [1] + [2] * n), d_first, d_fresh, i32(context), 2 * n + 1, 3, taps, heads, dim, second_at, span, 1e-6)
        if n > 1:
            ops.call(f"singe_conv_state_{ops.suffix}", stream(), rows, rows.stride(0), state, d_first, d_fresh, 2 * n + 1, 3, taps, span)
        assert (host(mixed)[n] == 0).all()
        for side, begin in ((0, 0), (1, n + 1)):
            mixed_all[side, at: at + n] = host(mixed)[begin: begin + n]
            inverse_all[side, at: at + n] = host(inverse)[begin: begin + n]
    for side in range(2):
        expect = ref.silu(ref.causal_convolution(projected[side].astype(np.float64), weight.T.astype(np.float64)))
        assert relative(mixed_all[side], expect) < LIMIT[dtype]
        for place, begin in ((0, 0), (1, second_at)):
            pieces = mixed_all[side][:, begin: begin + heads * dim].reshape(total, heads, dim)
            unit = pieces * inverse_all[side][:, place * heads: (place + 1) * heads, None]
            assert np.abs(unit - ref.unit(pieces)).max() < 1e-5


@pytest.mark.parametrize("taps", [1, 3, 4])
def test_convolution_over_a_long_ragged_prompt(taps):
    """Enough rows for tiles of several tokens: sequences end and begin inside tiles, some idle, some continue."""
    rng = np.random.default_rng(taps)
    ops, heads, dim, rest = Ops("bfloat16"), 3, 32, 40
    span = 2 * heads * dim + rest
    fresh = [700, 0, 1, 2, 3, 5, 0, 0, 1500, 9, 1, 1, 3000]
    context = [0, 5, 7, 0, 1, 2, 0, 9, 0, 4, 0, 1, 2]
    counts = [max(n, 1) for n in fresh]
    first, rows = np.cumsum([0] + counts)[:-1], sum(counts)
    past = [draw(rng, min(c, taps - 1), span) for c in context]
    projected, weight = draw(rng, rows, span), draw(rng, taps, span)
    state = torch.full((len(fresh), taps - 1, span), float("nan"), dtype=ops.dtype, device="cuda")
    for s, values in enumerate(past):
        if len(values):
            state[s, taps - 1 - len(values):] = dev(values).to(ops.dtype)
    mixed, inverse = ops.rows(rows, span), torch.empty((rows, 2 * heads), device="cuda")
    sequence_of = np.repeat(np.arange(len(fresh)), counts)
    d_projected, d_taps, d_first, d_fresh = ops.weight(projected), dev(weight).to(ops.dtype), i32(first), i32(fresh)
    ops.call("singe_conv_recurrence_inputs_bf16", stream(), mixed, mixed.stride(0), inverse, d_projected, d_projected.stride(0), d_taps, state,
             i32(sequence_of), d_first, d_fresh, i32(context), rows, len(fresh), taps, heads, dim, heads * dim, span, 1e-6)
    ops.call("singe_conv_state_bf16", stream(), d_projected, d_projected.stride(0), state, d_first, d_fresh, rows, len(fresh), taps, span)
    got, lengths, after = host(mixed), host(inverse), host(state)
    for s, n in enumerate(fresh):
        if n == 0:
            assert (got[first[s]] == 0).all()
            continue
        wide = np.concatenate([past[s], projected[first[s]: first[s] + n]])
        expect = ref.silu(ref.causal_convolution(wide.astype(np.float64), weight.T.astype(np.float64)))[len(past[s]):]
        part = got[first[s]: first[s] + n]
        assert relative(part, expect) < LIMIT["bfloat16"], f"sequence {s}"
        for place in range(2):
            pieces = part[:, place * heads * dim: (place + 1) * heads * dim].reshape(n, heads, dim)
            unit = pieces * lengths[first[s]: first[s] + n, place * heads: (place + 1) * heads, None]
            assert np.abs(unit - ref.unit(pieces)).max() < 1e-5
        kept = wide[max(len(wide) - taps + 1, 0):] if taps > 1 else wide[:0]
        assert np.array_equal(after[s, taps - 1 - len(kept):], kept), f"state of sequence {s}"


ROTATIONS = [{"dims": 16, "base": 10000.0}, {"dims": 24, "base": 500.0, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}},
             {"dims": 2, "base": 100.0, "scaling": {"factor": 1.0, "original": 4096, "fast": 32.0, "slow": 32.0}}]


def rotation_of(rot):
    return Rotation(rot["dims"], rot["base"], YarnScaling(**rot["scaling"]) if "scaling" in rot else None)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("rot", ROTATIONS)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,size,taps", [(6, 2, 40, 24, 64, 3), (2, 1, 25, 37, 40, 1), (3, 3, 128, 96, 128, 2)])
def test_attention_inputs(dtype, rot, heads, kv_heads, dim, vdim, size, taps):
    """Bias, convolution, norm over the whole projection, rotation at positions from 0 and from 100 000 on, the cache rows and
    the packed rows."""
    rng = np.random.default_rng(dim + taps)
    ops, tokens, page_size, eps = Ops(dtype), 23, 5, 1e-5
    widths = (heads * dim, kv_heads * dim, kv_heads * vdim)
    _, key_at, value_at, span = [0] + [int(v) for v in np.cumsum([round_up(w, 8) for w in widths])]
    u, bias, weight = draw(rng, tokens, span, scale=2.0), draw(rng, span), draw(rng, taps, span)
    norms = [draw(rng, heads * dim), draw(rng, kv_heads * dim)]
    rotation = rotation_of(rot)
    frequencies = torch.from_numpy(rotation.frequencies()).cuda()
    for start in (0, 100000):
        projected = ops.weight(u)
        state = torch.zeros((1, taps - 1, span), dtype=ops.dtype, device="cuda")
        before = draw(rng, max(taps - 1, 0), span) if start else np.zeros((0, span), dtype=np.float32)
        if start and taps > 1:
            state[0] = dev(before).to(ops.dtype)
        query = torch.full((tokens, heads * size), float("nan"), dtype=ops.dtype, device="cuda")
        caches = [torch.full((8, page_size, kv_heads * size), float("nan"), dtype=ops.dtype, device="cuda") for _ in range(2)]
        packed = [torch.full((40, kv_heads * size), float("nan"), dtype=ops.dtype, device="cuda") for _ in range(2)]
        pages, slots = rng.permutation(8)[np.arange(tokens) // page_size], np.arange(tokens) % page_size
        cached, packed_rows = (np.arange(tokens) % 3 != 0).astype(np.uint8), np.where(np.arange(tokens) % 4 == 1, -1, np.arange(tokens) + 9)
        status = torch.zeros(1, dtype=torch.int32, device="cuda")
        ops.call(f"singe_conv_attention_inputs_{ops.suffix}", stream(), query, query.stride(0), *caches, *packed, projected,
                 projected.stride(0), dev(bias).to(ops.dtype), dev(weight).to(ops.dtype), state, dev(norms[0]).to(ops.dtype),
                 dev(norms[1]).to(ops.dtype), frequencies, frequencies.numel(), rotation.magnitude(), i64(start + np.arange(tokens)),
                 i32([0] * tokens), i32([0]), i32([tokens]), i32([start]), i64(pages), i64(slots), dev(cached), i32(packed_rows), 40,
                 tokens, 1, taps, heads, kv_heads, dim, vdim, size, size, key_at, value_at, span, 8, page_size, eps, status)
        wide = np.concatenate([before, u]).astype(np.float64) + bias
        y = ref.causal_convolution(wide, weight.T.astype(np.float64))[len(before):]
        turn = lambda x, count: ref.rotate_adjacent(x.reshape(tokens, count, dim), start + np.arange(tokens, dtype=np.float64), rot)
        q = turn(ref.rms_norm(y[:, :widths[0]], norms[0], eps), heads)
        k = turn(ref.rms_norm(y[:, key_at: key_at + widths[1]], norms[1], eps), kv_heads)
        v = y[:, value_at: value_at + widths[2]].reshape(tokens, kv_heads, vdim)
        padded = lambda x: np.pad(x, ((0, 0), (0, 0), (0, size - x.shape[2])))
        assert relative(host(query).reshape(tokens, heads, size), padded(q)) < LIMIT[dtype]
        for cache, pack, expect in ((caches[0], packed[0], padded(k)), (caches[1], packed[1], padded(v))):
            got = host(cache).reshape(8, page_size, kv_heads, size)[pages, slots]
            assert relative(got[cached != 0], expect[cached != 0]) < LIMIT[dtype] and np.isnan(got[cached == 0]).all()
            rows = packed_rows[packed_rows >= 0]
            got = host(pack).reshape(40, kv_heads, size)
            assert relative(got[rows], expect[packed_rows >= 0]) < LIMIT[dtype]
            assert np.isnan(np.delete(got, rows, 0)).all()
        assert int(status.item()) == 0


# ---- attention within chunks ----

def one_key_stands_out(rng, tokens, kv_heads, size, target):
    """Keys of which the one at ``target`` answers a query of ones by far the most, and values that name their position."""
    key = draw(rng, tokens, kv_heads, size, scale=0.1)
    key[target] = 2.0
    return bf16(key), draw(rng, tokens, kv_heads, size)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("heads,kv_heads,size,page,chunk,splits", [
    (4, 2, 64, 16, 21, 1), (8, 1, 128, 16, 96, 2), (6, 3, 128, 16, 300, 5), (3, 1, 64, 16, 1, 1), (16, 2, 128, 16, 64, 3),
    (9, 1, 64, 16, 33, 1), (4, 2, 40, 16, 21, 1), (2, 2, 64, 1, 17, 1), (4, 1, 144, 64, 100, 1)])
def test_decode_attention_sees_its_own_chunk(dtype, heads, kv_heads, size, page, chunk, splits):
    """Queries just before, at and just after chunk and page edges; the key that stands out is the chunk's first, the last of the
    chunk before, the query's own or the next one."""
    rng = np.random.default_rng(chunk * size)
    ops = Ops(dtype)
    lens = sorted({n for n in (1, 2, chunk - 1, chunk, chunk + 1, 2 * chunk, 2 * chunk + 1, 2 * chunk + page, 3 * chunk - 1) if n > 0})
    stride = -(-(lens[-1] + 2) // page)
    total = stride * page
    queries, tables, keys, values, expects, row_lens = [], [], [], [], [], []
    for n in lens:
        begin = (n - 1) // chunk * chunk
        for target in {begin, begin - 1, n - 1, n, (begin + n) // 2}:
            if not 0 <= target < total:
                continue
            key, value = one_key_stands_out(rng, total, kv_heads, size, target)
            query = bf16(np.ones((1, heads, size)) + draw(rng, 1, heads, size, scale=0.1))
            expect = ref.chunked_attention(np.repeat(query, n - begin, 0).astype(np.float64), key[begin:n].astype(np.float64),
                                           value[begin:n].astype(np.float64), 4.0 / size, chunk)
            queries.append(query)
            keys.append(key)
            values.append(value)
            expects.append(expect[-1])
            row_lens.append(n)
    count = len(queries)
    order = rng.permutation(count * stride).reshape(count, stride)
    cache = lambda parts: np.concatenate(parts).reshape(count * stride, page, kv_heads, size)
    laid = lambda parts: dev(cache(parts)[np.argsort(order.reshape(-1))]).to(ops.dtype)
    # the last query has no key: its row becomes zeros
    query = np.concatenate(queries + [queries[0]])
    out = torch.full((count + 1, heads, size), float("nan"), dtype=ops.dtype, device="cuda")
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    operands = [dev(query).to(ops.dtype), laid(keys), laid(values), i32(list(range(count)) + [0]), i32(row_lens + [0]), i32(order),
                count + 1, heads, kv_heads, size, page, count * stride, count, stride, chunk]
    if dtype == "bfloat16":
        attn = torch.full((count + 1, heads, splits, size), float("nan"), device="cuda")
        lse = torch.full((count + 1, heads, splits), float("nan"), device="cuda")
        ops.call("singe_chunked_attention_bf16", stream(), out, attn, lse, *operands, splits, 4.0 / size, status)
    else:
        ops.call("singe_chunked_attention_f32", stream(), out, *operands, 4.0 / size, status)
    assert int(status.item()) == 0
    assert np.abs(host(out)[:-1] - np.stack(expects)).max() < (4e-2 if dtype == "bfloat16" else 2e-5)
    assert (host(out)[-1] == 0).all()


def test_decode_attention_reports_bad_rows():
    ops = Ops("bfloat16")
    cache = torch.zeros((4, 16, 1, 64), dtype=torch.bfloat16, device="cuda")
    query, out = torch.zeros((1, 1, 64), dtype=torch.bfloat16, device="cuda"), torch.zeros((1, 1, 64), dtype=torch.bfloat16, device="cuda")
    scratch = torch.zeros(1024, device="cuda")
    for sequence, length, page in ((5, 3, 0), (0, 200, 0), (0, 3, 9)):
        status = torch.zeros(1, dtype=torch.int32, device="cuda")
        ops.call("singe_chunked_attention_bf16", stream(), out, scratch, scratch, query, cache, cache, i32([sequence]), i32([length]),
                 i32([[page, 1]]), 1, 1, 1, 64, 16, 4, 1, 2, 32, 1, 1.0, status)
        assert int(status.item()) == ks.STATUS_INDEX_OUT_OF_BOUNDS


@pytest.mark.parametrize("heads,kv_heads,size", [(4, 2, 64), (6, 1, 128), (3, 3, 128)])
def test_prompt_attention_over_pieces_with_shared_keys(heads, kv_heads, size):
    """Pieces with keys before their queries, each a sequence of its own."""
    rng = np.random.default_rng(size + heads)
    fresh, lens = [1, 40, 128, 300, 17], [30, 40, 200, 300, 145]
    offsets_q, offsets_kv = np.cumsum([0] + fresh)[:-1], np.cumsum([0] + lens)[:-1]
    query, key, value = draw(rng, sum(fresh), heads, size), draw(rng, sum(lens), kv_heads, size), draw(rng, sum(lens), kv_heads, size)
    ops, scale = Ops("bfloat16"), 2.0 * size ** -0.5
    out = torch.zeros((sum(fresh), heads, size), dtype=torch.bfloat16, device="cuda")
    lse = torch.zeros((sum(fresh), heads), device="cuda")
    ops.call("singe_windowed_prefill_attention_bf16", stream(), out, lse, *[dev(x).to(torch.bfloat16) for x in (query, key, value)],
             kv_heads * size, i32(fresh), i32(lens), i32(offsets_q), i32(offsets_kv), None, 0, len(fresh), sum(fresh), sum(lens), heads,
             kv_heads, size, NO_WINDOW, scale)
    for n, m, q0, k0 in zip(fresh, lens, offsets_q, offsets_kv):
        padded = np.concatenate([np.zeros((m - n, heads, size)), query[q0: q0 + n]])
        expect = ref.chunked_attention(padded, key[k0: k0 + m].astype(np.float64), value[k0: k0 + m].astype(np.float64), scale, 1 << 20)
        assert np.abs(host(out)[q0: q0 + n] - expect[m - n:]).max() < 3e-2


def test_moved_rows_land_where_they_are_told():
    source = torch.arange(12 * 8, dtype=torch.float32, device="cuda").view(12, 8)
    out, status = torch.zeros((6, 8), device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
    call = lambda rows, targets: Ops("float32").call("singe_move_rows", stream(), out, source, i32(rows), i32(targets), 3, 32, 12, 6, status)
    call([11, 0, 4], [1, 5, 0])
    assert torch.equal(out[[1, 5, 0]], source[[11, 0, 4]]) and (out[[2, 3, 4]] == 0).all() and int(status.item()) == 0
    call([1, 2, 3], [2, 6, 3])
    assert int(status.item()) == ks.STATUS_INDEX_OUT_OF_BOUNDS


# ---- the gated delta rule ----

CASES = [  # heads, kv_heads, dim, vdim, log rate, bias, spread of the decays
    (4, 2, 24, 40, -1.0, 0.0, 1.0),
    (2, 2, 32, 32, 0.0, -2.0, 1.0),
    (3, 1, 128, 128, -2.0, 0.0, 1.0),
    (1, 1, 8, 8, 1.0, 0.0, 0.0),
    (2, 1, 256, 64, -3.0, 0.0, 1.0),
    (2, 2, 64, 264, -1.0, 0.0, 1.0),
    (4, 4, 64, 128, 3.0, 1.0, 2.0),     # decays too strong to factor
    (2, 1, 16, 80, 1.5, 0.0, 4.0),      # some blocks are, some are not
    (2, 1, 48, 96, -8.0, -4.0, 1.0),    # hardly any decay
]


class DeltaCase:
    def __init__(self, rng, counts, heads, kv_heads, dim, vdim, rate, bias, spread):
        self.sizes = heads, kv_heads, dim, vdim
        rows = int(sum(max(n, 1) for n in counts))
        self.first = np.cumsum([0] + [max(n, 1) for n in counts])[:-1]
        self.key_at = round_up(kv_heads * dim, 8)
        self.value_at = 2 * self.key_at
        self.columns = round_up(max(heads * dim, heads * vdim), 8)
        self.mixed = draw(rng, rows, self.value_at + round_up(heads * vdim, 8))
        # neighbouring tokens' keys resemble one another, so that the writes of a block interact, and every token's key its query,
        # so that no first read-out all but vanishes
        keys = self.mixed[:, self.key_at: self.value_at] * 0.7
        keys[1:] += keys[:-1].copy()
        keys[:, : kv_heads * dim] += 0.5 * self.mixed[:, : kv_heads * dim]
        self.mixed[:, self.key_at: self.value_at] = bf16(keys)
        self.strength, self.decay = draw(rng, rows, heads, scale=2.0), draw(rng, rows, 2 * self.columns, scale=spread)
        self.rate = (rate + 0.1 * rng.standard_normal(heads)).astype(np.float32)
        self.bias = (bias + 0.3 * rng.standard_normal(heads * dim)).astype(np.float32)
        self.norm = draw(rng, vdim)
        units = lambda at: self.mixed[:, at: at + kv_heads * dim].reshape(rows, kv_heads, dim).astype(np.float64)
        self.inverse = np.concatenate([1.0 / np.sqrt((units(at) ** 2).sum(2) + 1e-6) for at in (0, self.key_at)], 1).astype(np.float32)

    def operands(self, ops, out, state):
        d = lambda x: ops.weight(x)
        mixed, strength, decay = d(self.mixed), d(self.strength), d(self.decay)
        return [out, out.stride(0), mixed, mixed.stride(0), dev(self.inverse), strength, strength.stride(0), decay, decay.stride(0),
                dev(self.rate), dev(self.bias), dev(self.norm).to(ops.dtype), state]

    def expect(self, s, n, state, eps):
        heads, kv_heads, dim, vdim = self.sizes
        part = slice(self.first[s], self.first[s] + n)
        shared = np.arange(heads) // (heads // kv_heads)
        piece = lambda x, at, count, size: x[part, at: at + count * size].reshape(n, count, size).astype(np.float64)
        query = ref.unit(piece(self.mixed, 0, kv_heads, dim))[:, shared] * dim ** -0.5
        key = ref.unit(piece(self.mixed, self.key_at, kv_heads, dim))[:, shared]
        step = ref.softplus(piece(self.decay, 0, heads, dim) + self.bias.reshape(heads, dim))
        decay = np.exp(-np.exp(self.rate.astype(np.float64))[:, None] * step)
        out, state = ref.delta_recurrence(query, key, piece(self.mixed, self.value_at, heads, vdim), decay,
                                          ref.sigmoid(self.strength[part].astype(np.float64)), state)
        return ref.rms_norm(out, self.norm, eps) * ref.sigmoid(piece(self.decay, self.columns, heads, vdim)), state


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("case", CASES + [(2, 1, 10, 13, -1.0, 0.0, 1.0), (1, 1, 33, 300, -1.0, 0.0, 1.0), (1, 1, 300, 20, -1.0, 0.0, 1.0)])
def test_delta_rule_token_by_token(dtype, case):
    rng = np.random.default_rng(case[2] * case[3])
    counts, contexts, eps = [1, 0, 3, 7, 1, 4], [0, 5, 0, 4, 9, 1], 1e-6
    delta = DeltaCase(rng, counts, *case)
    heads, kv_heads, dim, vdim = delta.sizes
    before = draw(rng, 6, heads, dim, vdim, exact16=False)
    ops = Ops(dtype)
    state, out = dev(before), ops.rows(len(delta.mixed), heads * vdim)
    out.fill_(float("nan"))
    ops.call(f"singe_gated_delta_step_{ops.suffix}", stream(), *delta.operands(ops, out, state), i32(delta.first), i32(counts), i32(contexts),
             len(delta.mixed), 6, heads, kv_heads, dim, vdim, delta.key_at, delta.value_at, delta.columns, eps, 5)
    got, after = host(out).reshape(-1, heads, vdim), host(state)
    for s, n in enumerate(counts):
        first = delta.first[s]
        if n == 0:
            assert (got[first] == 0).all() and np.array_equal(after[s], before[s])
        elif n > 5:
            assert np.isnan(got[first: first + n]).all() and np.array_equal(after[s], before[s])
        else:
            expect, end = delta.expect(s, n, before[s].astype(np.float64) * (contexts[s] > 0), eps)
            assert relative(got[first: first + n], expect) < {"bfloat16": 6e-3, "float32": 1e-4}[dtype]
            assert relative(after[s], end) < 1e-5


@pytest.mark.parametrize("case,many", [(case, False) for case in CASES] + [(case, True) for case in CASES[2:7]])
def test_delta_rule_block_by_block(case, many):
    """``many``: enough sequences to fill the machine, so that a block's key tiles stay with one warp."""
    rng = np.random.default_rng(case[2] + case[3] + case[0])
    counts, contexts, eps = [16, 9, 1, 333, 15, 17, 600, 0], [0, 3, 7, 0, 0, 20, 5, 2], 1e-6
    if many:
        counts, contexts = [21] * 90 + [40], [0, 2, 0] * 30 + [5]
    delta = DeltaCase(rng, counts, *case)
    heads, kv_heads, dim, vdim = delta.sizes
    before = draw(rng, len(counts), heads, dim, vdim, exact16=False)
    served = [s for s, n in enumerate(counts) if n > 8]
    starts = [np.arange(delta.first[s], delta.first[s] + counts[s], 16) for s in served]
    tokens = np.concatenate([np.minimum(delta.first[s] + counts[s] - start, 16) for s, start in zip(served, starts)])
    blocks = [len(start) for start in starts]
    runs = np.stack([served, np.cumsum(blocks) - blocks, blocks], 1)
    ops, rows = Ops("bfloat16"), len(delta.mixed)
    state, out = dev(before), ops.rows(rows, heads * vdim)
    out.fill_(float("nan"))
    size = int(ks.lib().singe_gated_delta_prompt_scratch(heads, dim, vdim, rows, len(tokens)))
    assert size > 0
    scratch = torch.full((size,), 255, dtype=torch.uint8, device="cuda")
    ops.call("singe_gated_delta_prompt_bf16", stream(), *delta.operands(ops, out, state), i32(contexts), rows, heads, kv_heads, dim, vdim,
             delta.key_at, delta.value_at, delta.columns, eps, i32(np.concatenate(starts)), i32(tokens), len(tokens), i32(runs), len(runs),
             scratch)
    got, after = host(out).reshape(-1, heads, vdim), host(state)
    for s, n in enumerate(counts):
        first = delta.first[s]
        if s not in served:
            assert np.array_equal(after[s], before[s]) and np.isnan(got[first: first + max(n, 1)]).all()
            continue
        expect, end = delta.expect(s, n, before[s].astype(np.float64) * (contexts[s] > 0), eps)
        assert relative(got[first: first + n], expect) < 8e-3, f"sequence {s}"
        assert relative(after[s], end) < 1e-3, f"state of sequence {s}"   # one bf16 rounding would leave more
    assert ks.lib().singe_take_device_error(None) == 0


def test_gated_unit_in_32_bit():
    rng = np.random.default_rng(2)
    ops, x = Ops("float32"), draw(rng, 5, 20)
    gate, up = draw(rng, 33, 20), draw(rng, 33, 20)
    out = ops.rows(5, 33)
    ops.gated_linear_unit(stream(), out, ops.weight(x), ops.gate_up_weight(gate, up))
    assert relative(host(out), ref.silu(x.astype(np.float64) @ gate.T) * (x.astype(np.float64) @ up.T)) < 5e-6
