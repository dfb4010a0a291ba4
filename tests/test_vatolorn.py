"""Vatolorn, host side: configuration and checkpoint names, rotation frequencies, chunks in the page table, the pieces of a
prompt.  No GPU."""
import copy

import numpy as np
import pytest

from oracle import vatolorn_ref
from singe_b200 import checkpoint, models
from singe_b200.decoder import PageTable
from singe_b200.layer_ops import plan_chunks
from singe_b200.parallel_mixer import Rotation, YarnScaling, parts_at
from tests import vatolorn_util as util


def _read(tmp_path, config, weights=None):
    directory = util.write_snapshot(tmp_path, config, util.make_weights(config) if weights is None else weights)
    snapshot = checkpoint.Snapshot(directory)
    read = checkpoint.read_hybrid_config(directory, snapshot)
    checkpoint.check_keys(snapshot, checkpoint.hybrid_names(read))
    assert models.architecture(directory) == "Vatolorn"
    return read


@pytest.mark.parametrize("config", [util.MIXED, util.ODD, util.ONES, util.WIDE])
def test_every_size_and_constant_comes_from_the_files(tmp_path, config):
    read = _read(tmp_path, config)
    assert (read.width, read.vocab, read.eps, read.streams, read.logit_scale) == (
        config["width"], config["vocab"], config["norm"]["eps"], config["streams"], config["logit_scale"])
    for index, (layer, entry) in enumerate(zip(read.layers, config["layers"])):
        for got, want in ((layer.mixer.left, entry["mixer"]["left"]), (layer.mixer.right, entry["mixer"]["right"])):
            assert (got.heads, got.kv_heads, got.dim, got.vdim, got.taps) == tuple(
                want[name] for name in ("heads", "kv_heads", "dim", "vdim", "conv"))
        left, fields = layer.mixer.left, entry["mixer"]["left"]
        assert (left.chunk, left.scale) == (fields["mask"]["size"], fields["scale"])
        scaling = fields["rot"]["scaling"]
        assert left.rotation == Rotation(fields["rot"]["dims"], fields["rot"]["base"],
                                         YarnScaling(scaling["factor"], scaling["original"], scaling["fast"], scaling["slow"]))
        assert (layer.mixer.right.rank, layer.mixer.right.gate_rank) == (12 + index, 17 - 2 * index)
        assert layer.gated and layer.ffn == (entry["mlp"]["ff"] if entry["mlp"] else 0)
    assert read.chunks() == sorted({entry["mixer"]["left"]["mask"]["size"] for entry in config["layers"]}) and read.window() == 0


def test_what_the_decoder_would_pass_over_is_refused(tmp_path):
    def broken(change):
        config = copy.deepcopy(util.MIXED)
        weights = util.make_weights(config)
        change(config)
        with pytest.raises((checkpoint.UnsupportedConfig, checkpoint.CheckpointError)):
            _read(tmp_path, config, weights)

    side = lambda c, name: c["layers"][0]["mixer"][name]
    broken(lambda c: side(c, "left").update(sinks=2))
    broken(lambda c: side(c, "left")["mask"].update(keep=4))
    broken(lambda c: side(c, "left")["rot"].update(dims=41))
    broken(lambda c: side(c, "left")["rot"].update(dims=44))           # more than a head has
    broken(lambda c: side(c, "left")["rot"]["scaling"].update(factor=0.0))
    broken(lambda c: side(c, "left")["rot"]["scaling"].update(truncate=True))
    broken(lambda c: side(c, "left").update(kv_heads=4))               # six heads do not share four
    broken(lambda c: side(c, "right").update(tau=1.0))
    broken(lambda c: side(c, "right").update(conv=3))                  # a tensor of another shape
    broken(lambda c: c["layers"][0].update(type="attention"))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="experts"))
    broken(lambda c: c["layers"][1].update(mlp={"kind": "dense", "ff": 8}))
    broken(lambda c: c.pop("streams"))
    broken(lambda c: c.update(streams=2))
    broken(lambda c: c.update(tied=True))
    broken(lambda c: c.update(architecture="Kavalorn"))


@pytest.mark.parametrize("dims,base,scaling", [(64, 10000.0, (8.0, 1024, 32.0, 1.0)), (16, 500.0, (4.0, 64, 8.0, 1.0)), (2, 10.0, (1.0, 16, 1.0, 1.0)),
                                               (24, 1e6, (40.0, 4096, 32.0, 1.0)), (8, 100.0, None)])
def test_rotation_frequencies(dims, base, scaling):
    fields = None if scaling is None else dict(zip(("factor", "original", "fast", "slow"), scaling))
    rotation = Rotation(dims, base, None if scaling is None else YarnScaling(*scaling))
    frequency, factor = vatolorn_ref.yarn_frequencies(dims, base, fields)
    assert np.allclose(rotation.frequencies(), frequency, rtol=1e-12) and rotation.magnitude() == pytest.approx(factor)
    if scaling is None or scaling[0] == 1.0:
        assert np.allclose(frequency, base ** (-2.0 * np.arange(dims // 2) / dims))
    else:
        plain = base ** (-2.0 * np.arange(dims // 2) / dims)
        assert frequency[0] == plain[0] and np.all(frequency <= plain * (1 + 1e-12)) and np.all(frequency >= plain / scaling[0] * (1 - 1e-12))


def test_parts_start_at_multiples_of_eight():
    assert parts_at(3, 8, 17) == [0, 8, 16, 40]


@pytest.mark.parametrize("chunks,window,page", [((5,), 0, 4), ((21, 70), 0, 16), ((16,), 0, 16), ((1,), 0, 3), ((32,), 9, 4)])
def test_pages_of_chunks_left_behind_return_to_the_pool(chunks, window, page):
    rng = np.random.default_rng(sum(chunks) + page)
    capacity, widest = 200, max(chunks + (window,))
    table = PageTable.create_shared(2, capacity, page, 2 * (widest + 24 + 2 * page), window, chunks)
    for _ in range(30):
        counts = [int(rng.integers(0, 8)), int(rng.integers(0, 8))]
        if not any(counts) or max(l + n for l, n in zip(table.lengths, counts)) > capacity:
            continue
        before = list(table.lengths)
        step = table.step([[1] * n for n in counts])
        assert len(step.pages) == table.table_length()
        owned = [p for held in table.pages for p in held if p != table.scratch_page]
        assert len(owned) == len(set(owned)) and not set(owned) & set(table.free) and len(owned) + len(table.free) == table.pool
        for row, n in enumerate(counts):
            if n == 0:
                continue
            oldest = min([before[row] // size * size for size in chunks] + ([max(before[row] - window + 1, 0)] if window else []))
            for position in range(oldest, table.lengths[row]):
                assert table.pages[row][position // page] != table.scratch_page
            for place, held in enumerate(table.pages[row]):
                if (place + 1) * page <= oldest:
                    assert held == table.scratch_page


@pytest.mark.parametrize("size", [1, 7, 16, 50])
def test_pieces_of_a_prompt_cover_what_its_tokens_see(size):
    context, fresh = np.asarray([0, 13, 4, 50]), np.asarray([33, 40, 2, 0])
    first = np.asarray([0, 33, 73, 75])
    long = np.asarray([0, 1])
    plan = plan_chunks(size, context, fresh, first, long)
    key_of = {}   # packed row -> (sequence, position)
    for b in long:
        for i in range(fresh[b]):
            row = int(plan["packed"][first[b] + i])
            assert row not in key_of
            key_of[row] = (b, context[b] + i)
    for (b, position), row in zip(plan["moved"], plan["moved_to"]):
        assert row not in key_of and position < context[b]
        key_of[int(row)] = (b, position)
    assert sorted(key_of) == list(range(plan["keys"]))
    seen = set()
    for n, m, q0, k0 in zip(plan["lens_q"], plan["lens_kv"], plan["offsets_q"], plan["offsets_kv"]):
        for i in range(n):
            b = int(np.searchsorted(first, q0 + i, side="right") - 1)
            position = context[b] + (q0 + i - first[b])
            visible = [key_of[k0 + j] for j in range(m - n + i + 1)]
            assert visible == [(b, p) for p in range(position // size * size, position + 1)]
            seen.add(int(q0 + i))
    assert seen == set(range(73))
    assert (plan["packed"][73:] == -1).all() and (plan["cached"][73:] == 1).all()
    for b in long:
        end = context[b] + fresh[b]
        expect = np.arange(context[b], end) >= end // size * size
        assert np.array_equal(plan["cached"][first[b]: first[b] + fresh[b]] != 0, expect)
