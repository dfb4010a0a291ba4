"""The residual stream of a layer-list decoder, between its sublayers.

  ``LayerNormResidual``   one f32 stream; every sublayer reads its layer norm
  ``StreamResidual``      several f32 streams (hyper-connections): a sublayer reads a blend of them, RMS-normed, and its output
                          and a blend of the old streams make the new ones

Both take a sublayer's output in by the same launch that norms for the next one.
"""
from __future__ import annotations

from dataclasses import dataclass

from .layer_ops import Ops, round_up


@dataclass
class Sublayer:
    """Where a mixer or feed-forward joins the residual: its norm's weight, and with several streams its blends."""
    norm: object
    blend_in: object = None      # [streams]
    blend_out: object = None     # [streams]
    blend_mix: object = None     # [streams, streams], from and to
    output_norms: object = None  # weights of two outputs side by side whose normed mean is the sublayer's output


class LayerNormResidual:
    def __init__(self, config, take, ops: Ops):
        self.config, self.ops = config, ops
        self.embed = ops.torch.as_tensor(take("embed")).to("cuda").to(ops.dtype).contiguous()
        self.embed_norm, self.final = ops.weight(take("embed.norm")), ops.weight(take("final.norm"))

    def sublayer(self, take, prefix: str, number: int, output_norms=None) -> Sublayer:
        return Sublayer(self.ops.weight(take(f"{prefix}norm{number}")))

    def start(self, stream, rows, sublayer: Sublayer, normed, status):
        """The residual of a step's tokens, and what the first sublayer reads in ``normed``."""
        c = self.config
        residual = self.ops.torch.empty((rows.count, c.width), dtype=self.ops.torch.float32, device="cuda")
        self.ops.call(f"singe_embedding_layer_norm_{self.ops.suffix}", stream, residual, self.embed, rows.tokens, self.embed_norm,
                      rows.count, c.width, c.vocab, c.eps, status)
        self.ops.add_layer_norm(stream, residual, None, normed, sublayer.norm, c.eps)
        return residual

    def advance(self, stream, residual, delta, done: Sublayer, sublayer: Sublayer, normed) -> None:
        """Takes the output ``delta`` of ``done`` in and norms for ``sublayer``."""
        self.ops.add_layer_norm(stream, residual, delta, normed, sublayer.norm, self.config.eps)

    def finish(self, stream, residual, delta, done: Sublayer, normed) -> None:
        self.ops.add_layer_norm(stream, residual, delta, normed, self.final, self.config.eps)

    def peek(self, stream, residual, delta, done: Sublayer):
        """The residual with ``delta`` taken in, for inspection."""
        return residual + delta.float()


class StreamResidual:
    def __init__(self, config, take, ops: Ops):
        self.config, self.ops = config, ops
        self.embed = ops.torch.as_tensor(take("embed")).to("cuda").to(ops.dtype).contiguous()
        self.final = ops.weight(take("final.norm"))

    def sublayer(self, take, prefix: str, number: int, output_norms=None) -> Sublayer:
        scalars = lambda name: self.ops.scalars(take(f"{prefix}hc{number}.{name}"))
        return Sublayer(self.ops.weight(take(f"{prefix}norm{number}")), scalars("in"), scalars("out"), scalars("mix"), output_norms)

    def start(self, stream, rows, sublayer: Sublayer, normed, status):
        c, torch = self.config, self.ops.torch
        streams = torch.empty((rows.count, c.streams, c.width), dtype=torch.float32, device="cuda")
        self.ops.call(f"singe_stream_embedding_norm_{self.ops.suffix}", stream, streams, self.embed, rows.tokens,
                      sublayer.blend_in, normed, normed.stride(0), sublayer.norm, rows.count, c.streams, c.width, c.vocab, c.eps,
                      status)
        return streams

    def advance(self, stream, streams, delta, done: Sublayer, sublayer: Sublayer, normed) -> None:
        self._step(stream, streams, delta, done, sublayer.blend_in, 1, normed, sublayer.norm, 1.0)

    def finish(self, stream, streams, delta, done: Sublayer, normed) -> None:
        self._step(stream, streams, delta, done, None, 0, normed, self.final, self.config.logit_scale)

    def peek(self, stream, streams, delta, done: Sublayer):
        streams = streams.clone()
        self._step(stream, streams, delta, done, None, 1, None, None, 1.0)
        return streams.sum(1)

    def _step(self, stream, streams, delta, done: Sublayer, blend_in, store: int, normed, norm, scale: float) -> None:
        c = self.config
        left, right = done.output_norms or (None, None)
        self.ops.call(f"singe_stream_step_norm_{self.ops.suffix}", stream, streams, delta, delta.stride(0), 1 if left is None else 2,
                      round_up(c.width, 8), left, right, 0.5, done.blend_mix, done.blend_out, blend_in, store, normed,
                      0 if normed is None else normed.stride(0), norm, scale, streams.shape[0], c.streams, c.width, c.eps)
