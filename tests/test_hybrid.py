"""Layer-list decoder, host side: configuration and checkpoint names, the registry, windows in the page table, the
segments of a prompt, trace replay.  No GPU."""
import json

import numpy as np
import pytest

from oracle import hybrid_ref
from singe_b200 import checkpoint, models
from singe_b200.decoder import PageTable, PageTableError
from singe_b200.hybrid import GatedLinearConfig, HybridConfig, LatentAttentionConfig, LayerConfig, plan_segments
from singe_b200.trace import TraceReplay, replay
from tests import hybrid_util as util


def _read(tmp_path, config, weights=None):
    directory = util.write_snapshot(tmp_path, config, util.make_weights(config) if weights is None else weights)
    snapshot = checkpoint.Snapshot(directory)
    read = checkpoint.read_hybrid_config(directory, snapshot)
    checkpoint.check_keys(snapshot, checkpoint.hybrid_names(read))
    return read


@pytest.mark.parametrize("config", [util.MIXED, util.ODD, util.ONES, util.WIDE])
def test_every_size_and_constant_comes_from_the_files(tmp_path, config):
    read = _read(tmp_path, config)
    assert (read.width, read.vocab, read.eps) == (config["width"], config["vocab"], config["norm"]["eps"])
    assert len(read.layers) == len(config["layers"])
    for index, (layer, entry) in enumerate(zip(read.layers, config["layers"])):
        mixer = entry["mixer"]
        assert (layer.mixer.heads, layer.mixer.dim, layer.mixer.vdim) == (mixer["heads"], mixer["dim"], mixer["vdim"])
        if entry["type"] == "gla":
            assert isinstance(layer.mixer, GatedLinearConfig) and layer.mixer.tau == mixer["tau"]
            assert layer.mixer.rank == 12 + read.owner(index)   # the helper gives every layer its own rank
        else:
            assert isinstance(layer.mixer, LatentAttentionConfig)
            assert (layer.mixer.window, layer.mixer.scale) == (mixer["mask"]["size"], mixer["scale"])
            assert (layer.mixer.q_rank, layer.mixer.kv_rank) == (mixer["q_rank"], mixer["kv_rank"])
        assert layer.ffn == (entry["mlp"]["ff"] if entry["mlp"] else 0)
        assert layer.weights_of == entry.get("weights_of")


def test_what_the_decoder_would_pass_over_is_refused(tmp_path):
    def broken(change):
        config = util.variant(util.MIXED)
        weights = util.make_weights(config)
        change(config)
        with pytest.raises((checkpoint.UnsupportedConfig, checkpoint.CheckpointError)):
            _read(tmp_path, config, weights)

    broken(lambda c: c["layers"][1]["mixer"].update(rotary=64))
    broken(lambda c: c["layers"][1]["mixer"]["mask"].update(sinks=4))
    broken(lambda c: c["layers"][0].update(type="attention"))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="experts"))
    broken(lambda c: c["layers"][4].update(weights_of=4))
    broken(lambda c: c["layers"][4].update(weights_of=17))
    broken(lambda c: c["layers"][4].update(weights_of=2))            # another layer's sizes
    broken(lambda c: c["layers"][1]["mixer"].pop("scale"))
    broken(lambda c: c["layers"][2]["mixer"].update(kv_rank=71))     # a tensor of another shape
    broken(lambda c: c["layers"][1].update(mlp={"kind": "dense", "ff": 8}))   # tensors that are not there
    broken(lambda c: c["layers"][0]["mixer"].update(tau=0.0))


def test_borrowed_weights_are_followed_to_their_owner():
    mixer = GatedLinearConfig(1, 8, 8, 4, 2.0)
    config = HybridConfig(layers=[LayerConfig(mixer, 0, 2), LayerConfig(mixer, 0, 0), LayerConfig(mixer)])
    assert [config.owner(i) for i in range(3)] == [2, 2, 2]


def test_the_registry_reads_the_configuration(tmp_path):
    util.write_snapshot(tmp_path / "a", util.ONES, util.make_weights(util.ONES))
    assert models.architecture(str(tmp_path / "a")) == "Kavalorn"
    for name, fields in (("b", {"architectures": ["LlamaForCausalLM"]}), ("c", {"model_type": "llama"})):
        (tmp_path / name).mkdir()
        (tmp_path / name / "config.json").write_text(json.dumps(fields))
        assert models.architecture(str(tmp_path / name)) == "LlamaForCausalLM"
        with pytest.raises(checkpoint.UnsupportedConfig):
            models.load_decoder(str(tmp_path / name), 1, 16, dtype="float32")
    (tmp_path / "d").mkdir()
    (tmp_path / "d" / "config.json").write_text(json.dumps({"architecture": "Other"}))
    with pytest.raises(checkpoint.UnsupportedConfig):
        models.architecture(str(tmp_path / "d"))


# ---- pages that a window leaves behind ----

@pytest.mark.parametrize("window,page", [(1, 4), (5, 4), (8, 4), (9, 4), (17, 16), (3, 1)])
def test_pages_outside_every_window_return_to_the_pool(window, page):
    rng = np.random.default_rng(window * 100 + page)
    capacity = 200
    table = PageTable.create_shared(2, capacity, page, 2 * (window + 24 + 2 * page), window)
    for _ in range(30):
        portions = [int(rng.integers(0, 8)), int(rng.integers(0, 8))]
        if not any(portions) or max(l + n for l, n in zip(table.lengths, portions)) > capacity:
            continue
        before = list(table.lengths)
        step = table.step([[1] * n for n in portions])
        assert len(step.pages) == table.table_length()
        owned = [p for held in table.pages for p in held if p != table.scratch_page]
        assert len(owned) == len(set(owned)) and not set(owned) & set(table.free)
        assert len(owned) + len(table.free) == table.pool
        for row, n in enumerate(portions):
            if n == 0:
                continue
            # every key a token of this step sees is on a page of its own sequence
            for position in range(max(before[row] - window + 1, 0), table.lengths[row]):
                assert table.pages[row][position // page] != table.scratch_page
            # and a sequence never keeps a page that ended before its window
            for place, held in enumerate(table.pages[row]):
                if (place + 1) * page <= before[row] - window + 1:
                    assert held == table.scratch_page
    for row in range(2):
        table.release(row)
    assert sorted(table.free) == list(range(table.pool))


def test_a_step_without_pages_gives_nothing_back():
    table = PageTable.create_shared(1, 100, 4, 16, window=4)
    table.step([[1] * 12])
    pages, free = list(table.pages[0]), list(table.free)
    with pytest.raises(PageTableError):
        table.step([[1] * 30])
    assert (table.pages[0], table.free, table.lengths) == (pages, free, [12])
    table.step([[1] * 10])


# ---- segments ----

@pytest.mark.parametrize("blocks,heads", [([1], 1), ([40], 2), ([3, 90, 7], 4), ([200, 200], 16), ([5] * 50, 32)])
def test_segments_cover_every_block_once_in_order(blocks, heads):
    rows = plan_segments(blocks, heads, 148)
    covered, first = [], 0
    for place, count in enumerate(blocks):
        own = [row for row in rows if row[0] == place]
        assert [row[3] for row in own] == list(range(len(own)))
        assert [row[4] for row in own] == [0] * (len(own) - 1) + [1]
        covered += [block for row in own for block in range(row[1], row[1] + row[2])]
        first += count
    assert covered == list(range(sum(blocks)))
    if len(blocks) * heads >= 148:
        assert len(rows) == len(blocks)


# ---- trace replay ----

class FakeModel:
    """Logits of a token: (its sequence's row, how many tokens came before it, the token)."""

    def __init__(self, sequences):
        self.sequences, self.capacity = sequences, 64
        self.lengths = [0] * sequences
        self.status = np.zeros(1, dtype=np.int32)

    def reset(self):
        self.lengths = [0] * self.sequences

    def release(self, row):
        self.lengths[row] = 0

    def step_tokens(self, tokens, want=None):
        import torch

        rows = []
        for row, (new, places) in enumerate(zip(tokens, want)):
            rows += [[row, self.lengths[row] + place, new[place]] for place in places]
            self.lengths[row] += len(new)
        return torch.tensor(rows, dtype=torch.float32).reshape(len(rows), 3)


def test_trace_replay_orders_logits_by_entry_and_reuses_rows(tmp_path):
    lines = [json.dumps(step) for step in (
        {"step": 0, "entries": [{"id": "a", "tokens": [5, 6, 7], "want": [2, 0]}], "end": []},
        {"step": 1, "entries": [{"id": "b", "tokens": [8, 9], "want": [1]}, {"id": "a", "tokens": [4], "want": [0]}], "end": ["a"]},
        {"step": 2, "entries": [{"id": "c", "tokens": [3], "want": []}], "end": []},
        {"step": 3, "entries": [{"id": "c", "tokens": [2], "want": [0]}], "end": ["b", "c"]})]
    said = []
    replay(FakeModel(2), lines, str(tmp_path), said.append)
    assert said == [f"done {i}" for i in range(4)]
    read = lambda i: np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").reshape(-1, 3).tolist()
    assert read(0) == [[0, 2, 7], [0, 0, 5]]
    assert read(1) == [[1, 1, 9], [0, 3, 4]]
    assert not (tmp_path / "2.f32").exists()
    assert read(3) == [[0, 1, 2]]   # row 0 again, from its first position on


def test_trace_replay_refuses_more_requests_than_rows():
    state = TraceReplay(FakeModel(1))
    state.run({"step": 0, "entries": [{"id": "a", "tokens": [1]}], "end": []})
    with pytest.raises(ValueError, match="rows"):
        state.run({"step": 1, "entries": [{"id": "b", "tokens": [1]}], "end": []})


# ---- the oracle itself ----

def test_oracle_recurrence_is_the_sum_it_stands_for():
    rng = np.random.default_rng(0)
    t, h, k, v = 6, 2, 3, 4
    q, key, value = rng.standard_normal((t, h, k)), rng.standard_normal((t, h, k)), rng.standard_normal((t, h, v))
    decay = rng.uniform(0.2, 1.0, (t, h, k))
    out, _ = hybrid_ref.gated_recurrence(q, key, value, decay, np.zeros((h, k, v)))
    for i in range(t):
        expect = np.zeros((h, v))
        for j in range(i + 1):
            weight = (q[i] * key[j] * np.prod(decay[j + 1:i + 1], axis=0)).sum(axis=1)
            expect += weight[:, None] * value[j]
        assert np.allclose(out[i], expect)


def test_oracle_window_counts_the_token_itself():
    t = 7
    q, key = np.zeros((t, 1, 1)), np.zeros((t, 1, 1))
    value = np.arange(t, dtype=np.float64).reshape(t, 1, 1)
    out = hybrid_ref.windowed_attention(q, key, value, 1.0, 3)[:, 0, 0]
    assert np.allclose(out, [np.mean(range(max(0, i - 2), i + 1)) for i in range(t)])
