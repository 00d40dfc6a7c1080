"""How sublayers join a residual of several streams."""
from __future__ import annotations

import torch

from ..csrc import ops
from .base import Connection, ParamSpec, Streamed, register_part


@register_part("connection", "hyper")
class HyperConnection(Connection):
    """Learned static connection of a sublayer to s residual streams: with y the sublayer's output,
    X[j] <- sum_i mix[i, j] X[i] + out[j] y, all streams at once from the old ones (what the sublayer reads of the streams
    belongs to its norm, `streams_rmsnorm`).  mix, out: tensor names; the numbers are used in 32-bit."""

    graph_safe = True

    def __init__(self, streams: int, mix: str, out: str):
        if not 1 <= streams <= ops.MAX_STREAMS:
            raise ValueError(f"a residual has 1 to {ops.MAX_STREAMS} streams, got {streams}")
        self.streams, self.mix_name, self.out_name = int(streams), mix, out
        self.mix = self.out = None

    def params(self):
        return [ParamSpec(self.mix_name, (self.streams, self.streams), init="unit"),
                ParamSpec(self.out_name, (self.streams,), init="unit")]

    def bind(self, tensors, rt):
        self.mix, self.out = (tensors[n].to(torch.float32).contiguous() for n in (self.mix_name, self.out_name))

    def join(self, update) -> Streamed:
        return Streamed(update, self.mix, self.out)
