"""Token shift: what a mixer reads is moved, entry by entry, towards the row of the token before,

    out_t = h_t + (h_(t-1) - h_t) * share,      h = norm(x), h_(-1) = 0 for a sequence's first token.

The last token's h is state of the sequence (float32, in the layer's cache line behind the mixer's own state, twice: a step
that begins at position p reads copy p & 1 and writes copy (p + n) & 1).  h, the difference and the state are float32; only
the rows handed to the mixer are in the model dtype.  A norm that has ``forward_shifted`` runs norm and shift as one kernel
(``FIELDRUN_B200_FUSED_SHIFT=0``: two, for comparison); any other norm gives its float32 rows to a kernel of the shift alone."""
from __future__ import annotations

import os
from typing import Optional

import torch

from ..csrc import ops
from ..weights.loader import VECTOR, TensorNeed, TensorSource
from .base import MixerInput, register_part

FUSED_SHIFT = os.environ.get("FIELDRUN_B200_FUSED_SHIFT", "1") != "0"


class TokenShift(MixerInput):
    replayable = True

    def __init__(self, spec, dtype):
        super().__init__(spec, dtype)
        self.width = int(spec.args["width"])
        self.state_floats = self.width
        self.share: Optional[torch.Tensor] = None

    def tensor_needs(self):
        return [TensorNeed(self.name_of("share"), (self.width,), VECTOR, "around_half")]

    def load(self, source: TensorSource) -> None:
        self.share = source.fetch(self.tensor_needs()[0])

    def forward(self, ctx, norm, x, pending, line, offset):
        if FUSED_SHIFT and hasattr(norm, "forward_shifted"):
            return norm.forward_shifted(ctx, x, self.share, line.state, offset, delta=pending)
        _, h = norm.forward(ctx, x, delta=pending, want32=True)
        out = ctx.buffer(f"token_shift.out.{self.width}", tuple(h.shape), self.dtype)
        ops.token_shift(h, out, shift=(self.share, ctx, line.state, offset))
        return x, out


register_part("mixer_input", "token_shift", TokenShift, replace=True)
