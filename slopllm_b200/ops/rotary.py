"""Rotary frequency tables, made once on the host: plain and YaRN-scaled."""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional

import torch


@dataclass(frozen=True)
class YarnScaling:
    """Context extension by frequency interpolation: pairs that turn fewer than `slow` times over `original` positions are
    slowed down by `factor`, pairs that turn more than `fast` times keep their frequency, a linear ramp lies in between."""

    factor: float
    original: float
    fast: float
    slow: float


@dataclass
class RotaryTable:
    dims: int                 # rotated values at the front of the vector; value i pairs with value i + dims / 2
    freq: torch.Tensor        # fp32 [dims / 2]: angle per position
    gain: float               # factor on cos and sin

    def to(self, device) -> "RotaryTable":
        return RotaryTable(self.dims, self.freq.to(device), self.gain)

    def apply(self, x: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
        """fp32 rotate-half of the first `dims` values of x [T, ..., D] (the definition the kernels follow)."""
        xf, half = x.to(torch.float32), self.dims // 2
        ang = positions.to(torch.float32).unsqueeze(-1) * self.freq
        cos, sin = ang.cos() * self.gain, ang.sin() * self.gain
        while cos.dim() < xf.dim():
            cos, sin = cos.unsqueeze(1), sin.unsqueeze(1)
        a, b = xf[..., :half], xf[..., half:self.dims]
        return torch.cat([a * cos - b * sin, b * cos + a * sin, xf[..., self.dims:]], dim=-1)


def rotary_table(dims: int, base: float, yarn: Optional[YarnScaling] = None) -> RotaryTable:
    if dims % 2:
        raise ValueError("rotary dims must be even")
    inv = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if yarn is None:
        return RotaryTable(dims, torch.tensor(inv, dtype=torch.float32), 1.0)

    def pair_index(turns: float) -> float:       # the (real-valued) dimension whose pair makes `turns` turns over the original context
        return dims * math.log(yarn.original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    low = max(math.floor(pair_index(yarn.fast)), 0)
    high = min(math.ceil(pair_index(yarn.slow)), dims - 1)
    width = max(high - low, 0.001)
    freq = []
    for i, f in enumerate(inv):
        slowed = min(max((i - low) / width, 0.0), 1.0)
        freq.append(f * (1.0 - slowed) + f / yarn.factor * slowed)
    return RotaryTable(dims, torch.tensor(freq, dtype=torch.float32), 0.1 * math.log(yarn.factor) + 1.0)
