"""Replays a trace of given token ids through a decoder, step by step, and writes logits: no sampling.

Each line of the input is one step, ``{"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}``.  An entry's
tokens extend its request; ``want`` lists the places among them whose logits are written, in order, to ``<step>.f32``
(little-endian f32 rows of the vocabulary).  Requests in ``end`` give back what they hold once the step is done.
"""
from __future__ import annotations

import json
import os

import numpy as np

from .decoder import CachedDecoder


class TraceReplay:
    """The requests of a trace on the rows of a decoder."""

    def __init__(self, model):
        self.model = model
        self.decoder = CachedDecoder(model)
        self.decoder.reset()
        self.rows = {}
        self.free = list(range(self.decoder.sequences() - 1, -1, -1))

    def run(self, step: dict):
        """Runs one step; returns the wanted logits [wanted, vocab] as numpy, or None when nothing was wanted."""
        tokens = [[] for _ in range(self.decoder.sequences())]
        want = [[] for _ in tokens]
        order = []
        for entry in step.get("entries", []):
            request = entry["id"]
            if request not in self.rows:
                if not self.free:
                    raise ValueError(f"request {request}: all {len(tokens)} rows are taken")
                self.rows[request] = self.free.pop()
            row = self.rows[request]
            tokens[row] = entry["tokens"]
            want[row] = entry.get("want", [])
            order.append(row)
        logits = None
        if any(tokens):
            result = self.model.step_tokens(tokens, want=want)
            if any(want):
                # rows come in sequence order; the trace wants entry order
                starts = np.cumsum([0] + [len(places) for places in want])
                picked = [place for row in order for place in range(starts[row], starts[row + 1])]
                logits = result.float().cpu().numpy()[picked]
            self._verify()
        for request in step.get("end", []):
            row = self.rows.pop(request)
            self.decoder.release(row)
            self.free.append(row)
        return logits

    def _verify(self) -> None:
        status = int(self.model.status.item())
        if status != 0:
            raise RuntimeError(f"device status {status}")


def replay(model, lines, directory: str, report) -> None:
    """Runs every step of ``lines``; ``report(text)`` is called after each."""
    state = TraceReplay(model)
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = state.run(step)
        if logits is not None:
            logits.astype("<f4").tofile(os.path.join(directory, f"{step['step']}.f32"))
        report(f"done {step['step']}")
