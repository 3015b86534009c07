"""Retention: linear attention with one fixed decay per head, no softmax and no denominator.

Per head, with q and k of ``head_dim`` entries, v of ``value_dim`` and k multiplied by ``k_scale`` (head_dim^(-1/2)):

    S_t = decay_h S_(t-1) + k_t v_t^T,    o_t = S_t^T q_t

then each head's o_t is divided by its root mean square over ``value_dim`` (no weight), the heads side by side are
multiplied by silu(W_g x_t), and the output projection follows.  The state [heads, head_dim, value_dim] is float32, starts
at zero and lives twice in the cache line's state area (a step that begins at position p reads copy p & 1 and writes copy
(p + n) & 1).  q, k, v and the gate come from one product.

Kernels (retention.cu): the recurrence token by token in float32, for single tokens, float32 models and any sizes; and for
prompts in bfloat16 the same sums chunk by chunk on tensor cores: a chunk's own pairs as masked, decayed products of q and
k, what came before through the float32 state.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..cache import CacheNeed, LineView
from ..csrc import ops
from ..weights.loader import MATRIX, TensorNeed, TensorSource
from .base import Mixer, register_part
from .linear import linear

CHUNK_MIN_TOKENS = 8           # steps whose longest run of new tokens is shorter go token by token


class Retention(Mixer):
    replayable = True
    kernel_groups = ("common", "streams", "retention")

    def __init__(self, spec, dtype):
        super().__init__(spec, dtype)
        a = spec.args
        self.hidden_size = int(a["hidden_size"])
        self.num_heads = int(a["num_heads"])
        self.head_dim = int(a["head_dim"])
        self.value_dim = int(a.get("value_dim") or self.head_dim)
        self.k_scale = float(a.get("k_scale", self.head_dim ** -0.5))
        self.norm_eps = float(a.get("norm_eps", 1e-6))
        self.decay_values = tuple(float(d) for d in a["decay"])
        if min(self.num_heads, self.head_dim, self.value_dim) < 1:
            raise ValueError("retention needs heads, head_dim and value_dim of at least 1")
        if len(self.decay_values) != self.num_heads:
            raise ValueError(f"{len(self.decay_values)} decays for {self.num_heads} heads")
        if not ops.retention_takes(self.head_dim, self.value_dim):
            raise ValueError(f"a state of {self.head_dim} x {self.value_dim} per head is more than the retention kernel takes")
        self.qk_width = self.num_heads * self.head_dim
        self.v_width = self.num_heads * self.value_dim
        # columns of the one product in: q | k | v | gate, then zero rows up to a multiple of 16
        self.offsets = (0, self.qk_width, 2 * self.qk_width, 2 * self.qk_width + self.v_width)
        self.in_rows = -(-(2 * self.qk_width + 2 * self.v_width) // 16) * 16
        self.w_in: Optional[torch.Tensor] = None
        self.w_o: Optional[torch.Tensor] = None
        self.decay: Optional[torch.Tensor] = None

    def _needs(self) -> dict[str, TensorNeed]:
        d = self.hidden_size
        return {
            "q_proj": TensorNeed(self.name_of("q_proj"), (self.qk_width, d), MATRIX, "normal"),
            "k_proj": TensorNeed(self.name_of("k_proj"), (self.qk_width, d), MATRIX, "normal"),
            "v_proj": TensorNeed(self.name_of("v_proj"), (self.v_width, d), MATRIX, "normal"),
            "gate_proj": TensorNeed(self.name_of("gate_proj"), (self.v_width, d), MATRIX, "normal"),
            "o_proj": TensorNeed(self.name_of("o_proj"), (d, self.v_width), MATRIX, "normal"),
        }

    def tensor_needs(self):
        return list(self._needs().values())

    def load(self, source: TensorSource) -> None:
        needs = self._needs()
        stacked = [source.fetch(needs[n]) for n in ("q_proj", "k_proj", "v_proj", "gate_proj")]
        self.w_in = torch.zeros((self.in_rows, self.hidden_size), dtype=stacked[0].dtype, device=stacked[0].device)
        torch.cat(stacked, dim=0, out=self.w_in[:2 * self.qk_width + 2 * self.v_width])
        self.w_o = source.fetch(needs["o_proj"])

    def cache_need(self) -> CacheNeed:
        return CacheNeed(state_shape=(2, self.num_heads * self.head_dim * self.value_dim), state_dtype="float32")

    def prepare(self, num_positions: int, device) -> None:
        self.decay = ops.retention_decays(self.decay_values, device)

    def forward(self, ctx, act: torch.Tensor, line: LineView, writes_cache: bool) -> torch.Tensor:
        if not writes_cache:
            raise ValueError("a recurrent layer cannot read another layer's state: it has to write its own")
        rows = act.shape[0]
        # q | k | v | gate: float32 for the recurrence token by token; a bfloat16 prompt's chunks take them in bfloat16
        chunks = self.dtype == torch.bfloat16 and ctx.max_q_len >= CHUNK_MIN_TOKENS and ops.retention_chunks_take(self.head_dim, self.value_dim)
        proj = linear(act, self.w_in, rounded=chunks)                       # [T, in_rows]
        out = ctx.buffer("retention.out", (rows, self.v_width), self.dtype)
        raw = ctx.buffer("retention.raw", (rows, self.v_width), torch.float32)      # for steps that cut the heads over blocks
        ops.retention(proj, self.offsets, self.decay, ctx, line.state, 0, out, raw, heads=self.num_heads, dim=self.head_dim,
                      vdim=self.value_dim, k_scale=self.k_scale, eps=self.norm_eps)
        return linear(out, self.w_o)


register_part("mixer", "retention", Retention, replace=True)
