"""The Vatolorn decoder end to end: loader, steps of every shape, caches and states that are used again, generation, trace
replay -- against the plain float64 restatement in ``oracle.vatolorn_ref``."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracle import vatolorn_ref
from singe_b200 import layer_ops, models
from singe_b200.decoder import CachedDecoder, PageTableError
from singe_b200.generation import GenerationOptions, PromptChunks, RunningBatch, generate_batch
from tests import vatolorn_util as util
from tests.conftest import ROOT
from tests.decoder_checks import Expect, check, greedy, run_portions, small_pages, tokens_of

pytestmark = pytest.mark.gpu

CONFIGS = {"mixed": util.MIXED, "odd": util.ODD, "ones": util.ONES, "wide": util.WIDE}
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module")
def snapshots(tmp_path_factory):
    made = {}
    for name, config in CONFIGS.items():
        weights = util.make_weights(config, seed=len(name))
        made[name] = (config, weights, util.write_snapshot(tmp_path_factory.mktemp(name), config, weights))
    return made


@pytest.fixture(scope="module")
def expects(snapshots):
    return {name: Expect(vatolorn_ref, config, weights) for name, (config, weights, _) in snapshots.items()}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,length", [("mixed", 180), ("odd", 90), ("ones", 40), ("wide", 420)])
def test_whole_prompts_and_every_layer(snapshots, name, length, dtype):
    config, weights, directory = snapshots[name]
    decoder = models.load_decoder(directory, 1, 512, dtype)
    decoder.trail = []
    tokens = tokens_of(config, 1, length)
    logits = run_portions(decoder, 0, tokens, [length])
    expect, trail = vatolorn_ref.forward(config, weights, tokens)
    assert len(decoder.trail) == len(config["layers"])
    for index, residual in enumerate(decoder.trail):
        check(residual, trail[index], dtype, f"layer {index}")
    check(logits, expect, dtype, "logits")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,length", [("mixed", 150), ("odd", 70), ("ones", 30), ("wide", 40)])
def test_token_by_token_equals_the_prompt(snapshots, expects, name, length, dtype):
    config, _, directory = snapshots[name]
    decoder = models.load_decoder(directory, 2, 256, dtype)
    decoder.capture()
    tokens = tokens_of(config, 2, length)
    check(run_portions(decoder, 1, tokens, [1] * length), expects[name](tokens), dtype, "decoded from the first token")
    decoder.release(1)
    check(run_portions(decoder, 0, tokens, [length // 2] + [1] * (length - length // 2)), expects[name](tokens), dtype,
          "prompt, then decoded")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("portion", [2, 3, 7, 8, 9, 16, 17, 21, 22, 64, 70, 71])
def test_portions_of_every_size(snapshots, expects, portion, dtype):
    """Chunks of 21 and 70 tokens, pages of 16: portions end inside, at and just past the edges of each."""
    config, _, directory = snapshots["mixed"]
    decoder = models.load_decoder(directory, 1, 256, dtype)
    tokens = tokens_of(config, 3, 181)
    check(run_portions(decoder, 0, tokens, [portion] * (-(-len(tokens) // portion))), expects["mixed"](tokens), dtype,
          f"portions of {portion}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,portions", [("wide", [2, 64, 1, 129, 3, 8, 9, 128, 1, 1, 60, 24]), ("odd", [3, 1, 40, 2, 9, 1, 8, 26]),
                                           ("ones", [2, 3, 1, 20, 9])])
def test_portions_of_changing_size(snapshots, expects, name, portions, dtype):
    config, _, directory = snapshots[name]
    decoder = models.load_decoder(directory, 1, 512, dtype)
    tokens = tokens_of(config, 4, sum(portions))
    check(run_portions(decoder, 0, tokens, portions), expects[name](tokens), dtype, "portions")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_batches_of_unequal_requests_equal_each_alone(snapshots, expects, name, dtype):
    config, _, directory = snapshots[name]
    decoder = models.load_decoder(directory, 5, 256, dtype)
    requests = [tokens_of(config, 10 + i, n) for i, n in enumerate((120, 1, 33, 77, 64))]
    plans = [[50, 1, 1, 30, 8, 29, 1], [0, 0, 1, 0, 0, 0, 0], [1, 1, 1, 9, 1, 19, 1], [9, 8, 60, 0, 0, 0, 0], [0, 64, 0, 0, 0, 0, 0]]
    at, outs = [0] * 5, [[] for _ in range(5)]
    for index in range(7):
        parts = [request[a: a + plan[index]] for request, a, plan in zip(requests, at, plans)]
        logits = decoder.step_tokens(parts, want=[list(range(len(part))) for part in parts]).clone()
        counts = np.cumsum([0] + [len(part) for part in parts])
        for row in range(5):
            outs[row].append(logits[counts[row]: counts[row + 1]])
            at[row] += len(parts[row])
    assert int(decoder.status.item()) == 0
    for row, request in enumerate(requests):
        check(torch.cat(outs[row]), expects[name](request[: at[row]]), dtype, f"request {row}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("page_size", [16, 4])
def test_freed_pages_and_rows_are_used_again(snapshots, expects, page_size, dtype):
    """A pool just large enough for the chunks: pages move between sequences all the time, and a row's states start over with
    its next request."""
    config, _, directory = snapshots["mixed"]
    decoder = small_pages(directory, 2, 400, dtype, 2 * (70 + 64 + 32), page_size)
    decoder.capture()
    long = tokens_of(config, 20, 330)
    outs, at = [], 0
    other, other_at, other_outs, finished = tokens_of(config, 21, 50), 0, [], 0
    while at < len(long):
        n = (64, 1, 1, 20, 1, 3)[len(outs) % 6]
        part, spare = long[at: at + n], other[other_at: other_at + (1 if n == 1 else 16)]
        logits = decoder.step_tokens([part, spare], want=[range(len(part)), range(len(spare))]).clone()
        outs.append(logits[: len(part)])
        other_outs.append(logits[len(part):])
        at += len(part)
        other_at += len(spare)
        if other_at == len(other):
            check(torch.cat(other_outs), expects["mixed"](other), dtype, "short-lived request")
            decoder.release(1)
            finished += 1
            other, other_at, other_outs = tokens_of(config, 22 + finished % 2, 40), 0, []
    assert finished >= 3 and int(decoder.status.item()) == 0
    check(torch.cat(outs), expects["mixed"](long), dtype, "long request")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(snapshots, expects, dtype):
    config, _, directory = snapshots["mixed"]
    decoder = small_pages(directory, 1, 500, dtype, 112)
    decoder.capture()
    tokens = tokens_of(config, 5, 430)
    check(run_portions(decoder, 0, tokens, [9] + [1] * 421), expects["mixed"](tokens), dtype, "long decoding")


def test_a_chunk_is_left_behind_at_its_edge(snapshots, expects):
    """One layer, soft attention, no recurrence: the logits change with a token exactly as long as its chunk lasts."""
    config = util.model(64, 50, 2, 1.0, 1e-6, util.layer(util.left(2, 1, 16, 16, 24, 1, util.rot(2, 10.0, (1.0, 16, 1.0, 1.0)), 0.2),
                                                         util.right(1, 1, 8, 8, 1)))
    weights = util.make_weights(config, seed=9)
    weights["l0.mix.right.v"][:] = 0.0   # the recurrence carries nothing
    base = tokens_of(config, 7, 60)
    for dtype in DTYPES:
        for target in (23, 24, 47):
            other = list(base)
            other[target] = (base[target] + 17) % 50
            outs = []
            for tokens in (base, other):
                directory = util.write_snapshot(os.path.join(str(snapshots["mixed"][2]), "edge"), config, weights)
                decoder = models.load_decoder(directory, 1, 64, dtype)
                outs.append(run_portions(decoder, 0, tokens, [30] + [1] * 10 + [20]))
                check(outs[-1], vatolorn_ref.forward(config, weights, tokens)[0], dtype, f"target {target}")
            changed = ((outs[0] - outs[1]).abs().amax(1) > 1e-5).tolist()
            last = (target // 24 + 1) * 24
            assert not any(changed[:target]) and not any(changed[last:])
            assert all(changed[target:last]) if dtype == "float32" else changed[target]


def test_a_step_without_room_changes_nothing(snapshots, expects):
    config, _, directory = snapshots["mixed"]
    decoder = small_pages(directory, 2, 128, "float32", 96)
    tokens = tokens_of(config, 6, 60)
    first = run_portions(decoder, 0, tokens[:40], [40])
    with pytest.raises(PageTableError):
        decoder.step_tokens([tokens[40:], [1] * 60])
    with pytest.raises(PageTableError):
        decoder.step_tokens([[1] * 100, []])
    rest = run_portions(decoder, 0, tokens[40:], [20])
    check(torch.cat([first, rest]), expects["mixed"](tokens), "float32", "around a refused step")


def test_greedy_generation_through_the_scheduler(snapshots, expects):
    """Requests of unequal lengths join and leave a running batch of two rows, prompts in chunks."""
    config, _, directory = snapshots["mixed"]
    decoder = models.load_decoder(directory, 2, 256, "float32")
    decoder.capture()
    prompts = [tokens_of(config, 30 + i, n) for i, n in enumerate((70, 3, 41, 1))]
    batch = RunningBatch.create(CachedDecoder(decoder, PromptChunks(16, 16)), GenerationOptions(6))
    waiting, got = list(prompts), {}
    while waiting or not batch.is_empty():
        while waiting and (joined := batch.join(waiting[0])) is not None:
            got[joined] = []
            waiting.pop(0)
        for token in batch.advance():
            got[token.sequence].append(token.token)
    assert [got[i] for i in range(4)] == [greedy(expects["mixed"], prompt, 6) for prompt in prompts]
    assert generate_batch(CachedDecoder(decoder), prompts[:2], GenerationOptions(4)) == [got[0][:4], got[1][:4]]


def test_command_line_generates(snapshots, expects):
    config, _, directory = snapshots["mixed"]
    prompts = [tokens_of(config, 50, 20), tokens_of(config, 51, 5)]
    command = [sys.executable, "-m", "singe_b200", "generate", "--model", directory, "--dtype", "float32",
               "--max-new-tokens", "5"] + [part for prompt in prompts for part in ("--prompt", ",".join(map(str, prompt)))]
    result = subprocess.run(command, capture_output=True, text=True, cwd=ROOT, timeout=300)
    assert result.returncode == 0, result.stderr[-2000:]
    lines = [[int(t) for t in line.split(",")] for line in result.stdout.split()]
    assert lines == [greedy(expects["mixed"], prompt, 5) for prompt in prompts]


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_runner(snapshots, expects, tmp_path, dtype):
    config, _, directory = snapshots["odd"]
    first, second = tokens_of(config, 60, 60), tokens_of(config, 61, 30)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": first[:40], "want": [0, 39, 21]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": first[40:42], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": first[42:], "want": [17]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": second, "want": [29, 0]}], "end": ["y"]}]
    result = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", directory, "--dtype", dtype, "--out",
                             str(tmp_path), "--max-tokens", "64"], input="\n".join(map(json.dumps, steps)) + "\n",
                            capture_output=True, text=True, timeout=300)
    assert result.returncode == 0, result.stderr[-2000:]
    assert result.stdout.split("\n")[:4] == [f"done {i}" for i in range(4)]
    read = lambda i: torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").reshape(-1, config["vocab"]))
    check(read(0), expects["odd"](first)[[0, 39, 21]], dtype, "step 0")
    check(read(2), expects["odd"](first)[[59]], dtype, "step 2")
    check(read(3), expects["odd"](second)[[29, 0]], dtype, "step 3")


def test_prompts_and_short_portions_take_the_kernels_meant_for_them(snapshots, monkeypatch):
    """bf16 steps: the tensor-core prompt kernels for sizes they take."""
    called = set()
    original = layer_ops.Ops.call

    def record(self, name, *arguments):
        called.add(name)
        original(self, name, *arguments)

    monkeypatch.setattr(layer_ops.Ops, "call", record)
    tiled = {"singe_windowed_prefill_attention_bf16", "singe_gated_delta_prompt_bf16", "singe_chunked_attention_bf16",
             "singe_gated_delta_step_bf16"}
    config, _, directory = snapshots["mixed"]
    decoder = models.load_decoder(directory, 2, 64)
    called.clear()
    decoder.step_tokens([tokens_of(config, 1, 40), [1, 2]])
    assert tiled <= called
    called.clear()
    decoder.step_tokens([[3], [1, 2]])
    assert not called & {"singe_windowed_prefill_attention_bf16", "singe_gated_delta_prompt_bf16"}
