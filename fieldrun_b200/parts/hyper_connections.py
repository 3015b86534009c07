"""Hyper-connections: the residual stream is kept as S copies of a row, and a layer's sublayers read weighted sums of them.

A sublayer q has the constants in_q [S], out_q [S] and mix_q [S, S] (indexed [from, to]).  With y its output,

    it reads  u = sum_s in_q[s] x_s,   and then   x_t <- sum_s mix_q[s, t] x_s + out_q[t] y   for all copies at once.

A layer's two updates are linear in the copies and in both outputs, so they can be done in one step behind the layer:

    x_t <- sum_s (mix_1 mix_2)[s, t] x_s + (mix_2^T out_1)[t] y_1 + out_2[t] y_2

``load`` makes those products once, in float64, rounded to float32."""
from __future__ import annotations

from typing import Optional

import torch

from ..csrc import ops
from ..weights.loader import VECTOR, TensorNeed, TensorSource
from .base import StreamConnection, register_part


class HyperConnections(StreamConnection):
    """``streams`` copies; ``feed_forward`` False for a layer whose only sublayer is its mixer."""

    replayable = True
    kernel_groups = ("common", "copies")

    def __init__(self, spec, dtype):
        super().__init__(spec, dtype)
        self.streams = int(spec.args["streams"])
        self.feed_forward = bool(spec.args.get("feed_forward", True))
        if not 1 <= self.streams <= ops.STREAM_COPIES:
            raise ValueError(f"{self.streams} copies of the stream are outside 1..{ops.STREAM_COPIES}")
        self.gather1: Optional[torch.Tensor] = None
        self.gather2: Optional[torch.Tensor] = None
        self.out1: Optional[torch.Tensor] = None
        self.out2: Optional[torch.Tensor] = None
        self.mix1: Optional[torch.Tensor] = None
        self.mix_both: Optional[torch.Tensor] = None
        self.out1_through: Optional[torch.Tensor] = None      # out1 after the second mix

    def _needs(self, sublayer: int):
        s = self.streams
        return (TensorNeed(self.name_of(f"in{sublayer}"), (s,), VECTOR, "around_half"),
                TensorNeed(self.name_of(f"out{sublayer}"), (s,), VECTOR, "around_one"),
                TensorNeed(self.name_of(f"mix{sublayer}"), (s, s), VECTOR, "near_identity"))

    def tensor_needs(self):
        return [need for sublayer in ((1, 2) if self.feed_forward else (1,)) for need in self._needs(sublayer)]

    def load(self, source: TensorSource) -> None:
        self.gather1, self.out1, self.mix1 = (source.fetch(need) for need in self._needs(1))
        if self.feed_forward:
            self.gather2, self.out2, mix2 = (source.fetch(need) for need in self._needs(2))
            self.mix_both = (self.mix1.double() @ mix2.double()).to(torch.float32).contiguous()
            self.out1_through = (self.out1.double() @ mix2.double()).to(torch.float32).contiguous()


register_part("stream_connection", "hyper_connections", HyperConnections, replace=True)
