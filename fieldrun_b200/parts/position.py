"""Rotary position encoding as tables of cos and sin over positions.

The angle of pair j at position p is p * theta^(-2j / rotary_dim), j < rotary_dim/2
(src/minimax.rs:50,76 with rotary_dim = head_dim; the partial form with
rotary_dim < head_dim is src/qwen35moe.rs:78-81,121-138).  The reference forms
the angle and its cos/sin in float32 for every element; here the table is
computed once on the host in float64 and rounded to float32, which is at least
as close to the exact angle.  ``pairing`` "half" rotates (j, j + rotary_dim/2) as
the reference does; "interleaved" rotates (2j, 2j+1).

``frequency_blend`` {factor, low, high, original} changes the frequencies f_j by their wavelengths 2 pi / f_j: those below
original / high stay, those above original / low are divided by factor, and one in between, at
s = (original / wavelength - low) / (high - low), becomes (1 - s) f / factor + s f.
"""
from __future__ import annotations

import math

import torch

from .base import Position, register_part


class Rotary(Position):
    def __init__(self, args):
        self.rotary_dim = int(args["rotary_dim"])
        self.theta = float(args["theta"])
        pairing = args.get("pairing", "half")
        if pairing not in ("half", "interleaved"):
            raise ValueError(f"rotary pairing {pairing!r} is neither 'half' nor 'interleaved'")
        if self.rotary_dim % 2:
            raise ValueError(f"rotary_dim {self.rotary_dim} must be even")
        self.interleaved = pairing == "interleaved"
        self.position_scale = float(args.get("position_scale", 1.0))
        blend = args.get("frequency_blend")
        self.blend = tuple(float(blend[name]) for name in ("factor", "low", "high", "original")) if blend else None
        if self.blend is not None and not (self.blend[0] > 0.0 and 0.0 < self.blend[1] <= self.blend[2] and self.blend[3] > 0.0):
            raise ValueError(f"a frequency blend of (factor, low, high, original) = {self.blend}")

    def frequencies(self) -> torch.Tensor:
        """float64 [rotary_dim / 2]: the angle of every pair at position 1."""
        j = torch.arange(self.rotary_dim // 2, dtype=torch.float64)
        inv = 1.0 / torch.pow(torch.tensor(self.theta, dtype=torch.float64), 2.0 * j / self.rotary_dim)
        if self.blend is None:
            return inv
        factor, low, high, original = self.blend
        wavelength = 2.0 * math.pi / inv
        share = (original / wavelength - low) / max(high - low, 1e-300)        # high == low: no wavelength lies in between
        between = (1.0 - share) * inv / factor + share * inv
        return torch.where(wavelength < original / high, inv, torch.where(wavelength > original / low, inv / factor, between))

    def tables(self, num_positions: int, device):
        half = self.rotary_dim // 2
        if half == 0:
            return None, None
        inv = self.frequencies()
        pos = torch.arange(num_positions, dtype=torch.float64) * self.position_scale
        angle = pos[:, None] * inv[None, :]
        return (torch.cos(angle).to(torch.float32).to(device).contiguous(),
                torch.sin(angle).to(torch.float32).to(device).contiguous())


register_part("position", "rotary", Rotary, replace=True)
