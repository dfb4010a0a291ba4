"""What the whole-decoder tests share: comparison with an oracle's logits, stepping a request in portions, greedy decoding by an
oracle."""
import numpy as np
import torch

from singe_b200 import hybrid
from singe_b200.checkpoint import load_hybrid

# root mean square of a position's logit error over that of its logits
LIMIT = {"float32": 3e-5, "bfloat16": 6e-2}


class Expect:
    """Oracle logits of whole sequences, computed once each."""

    def __init__(self, oracle, config, weights):
        self.oracle, self.config, self.weights, self.known = oracle, config, weights, {}

    def __call__(self, tokens):
        key = tuple(tokens)
        if key not in self.known:
            self.known[key] = self.oracle.forward(self.config, self.weights, tokens)[0]
        return self.known[key]


def small_pages(directory, sequences, capacity, dtype, cache_tokens, page_size=16):
    """A decoder with small cache pages, so that a small pool still has pages to move around."""
    config, weights = load_hybrid(directory)
    config.page_size = page_size
    return hybrid.HybridDecoder(config, sequences, capacity, weights, dtype, cache_tokens)


def tokens_of(config, seed, count):
    return [int(t) for t in np.random.default_rng(seed).integers(0, config["vocab"], size=count)]


def check(got, expect, dtype, what):
    got, expect = got.float().cpu().numpy().astype(np.float64), np.asarray(expect)
    error = np.sqrt(((got - expect) ** 2).mean(1) / (expect ** 2).mean(1))
    assert np.isfinite(got).all(), what
    assert error.max() < LIMIT[dtype], f"{what}: position {error.argmax()} of {len(error)}: {error.max():.2e}"


def run_portions(decoder, row, tokens, portions):
    """Steps one row through ``tokens`` in portions, everything wanted; returns all logits."""
    outs, at = [], 0
    for n in portions:
        part, want = [[] for _ in range(decoder.sequences)], [[] for _ in range(decoder.sequences)]
        part[row], want[row] = tokens[at: at + n], list(range(len(tokens[at: at + n])))
        outs.append(decoder.step_tokens(part, want=want).clone())
        at += n
    assert at >= len(tokens) and int(decoder.status.item()) == 0
    return torch.cat(outs)


def greedy(expect, prompt, count):
    tokens = list(prompt)
    for _ in range(count):
        tokens.append(int(expect(tokens)[-1].argmax()))
    return tokens[len(prompt):]
