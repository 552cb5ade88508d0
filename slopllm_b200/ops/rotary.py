"""Rotary frequency tables, made once on the host: plain and YaRN-scaled; tables of angles that the layers of a model share."""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

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


# ---- angles shared by all layers of a step --------------------------------------------------------------------------------

def adjacent_order(size: int, dims: int) -> torch.Tensor:
    """Order of a head's values that puts the partners i and i + dims/2 of a rotate-half rotation side by side: place 2i holds value
    i, place 2i + 1 value i + dims/2, the values behind `dims` stay.  A projection whose rows are stored in this order needs no
    shuffling at run time; whatever reads its result in the same order (keys against queries, the output projection's columns)
    gives the same sums."""
    half = torch.arange(dims // 2)
    return torch.cat([torch.stack([half, half + dims // 2], 1).reshape(-1), torch.arange(dims, size)])


@dataclass(frozen=True)
class Turn:
    """A rotation of adjacent pairs: the first `dims` values of a vector, angles at columns `at` .. of the model's table."""

    dims: int
    at: int

    def columns(self, angles: torch.Tensor) -> torch.Tensor:
        return angles[:, self.at:self.at + self.dims // 2]

    def apply(self, x: torch.Tensor, angles: torch.Tensor, back: bool = False) -> torch.Tensor:
        """fp32 x [T, ..., D] turned by its token's angles, or back (the definition the kernels follow)."""
        xf, cs = x.to(torch.float32), self.columns(angles)
        cos, sin = cs[..., 0], -cs[..., 1] if back else cs[..., 1]
        while cos.dim() < xf.dim():
            cos, sin = cos.unsqueeze(1), sin.unsqueeze(1)
        a, b = xf[..., 0:self.dims:2], xf[..., 1:self.dims:2]
        pairs = torch.stack([a * cos - b * sin, b * cos + a * sin], -1).flatten(-2)
        return torch.cat([pairs, xf[..., self.dims:]], -1)


class AngleTable:
    """Cosines and sines of a step's positions for every rotation that some layer of a model uses, fp32 [T, pairs, 2]; made once a
    step (`csrc/rotary.cu`)."""

    def __init__(self):
        self._freq: List[float] = []
        self._turns: Dict[Tuple[int, float], Turn] = {}
        self._dev: Optional[torch.Tensor] = None

    def turn(self, dims: int, base: float) -> Turn:
        """The rotation with angles position * base^(-2i/dims); equal ones share their columns."""
        if dims % 2:
            raise ValueError("rotary dims must be even")
        key = (int(dims), float(base))
        if key not in self._turns:
            self._turns[key] = Turn(int(dims), len(self._freq))
            self._freq += [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
        return self._turns[key]

    def of(self, st) -> torch.Tensor:
        """The table of a step's positions (kept in the step's state)."""
        a = st.extra.get("angles")
        if a is None:
            a = st.extra["angles"] = self.at(st.positions)
        return a

    def at(self, positions: torch.Tensor) -> torch.Tensor:
        if self._dev is None or self._dev.device != positions.device:
            self._dev = torch.tensor(self._freq, dtype=torch.float64, device=positions.device)
        T, n = positions.shape[0], len(self._freq)
        if positions.is_cuda:
            from . import native as N
            out = torch.empty(T, n, 2, dtype=torch.float32, device=positions.device)
            N.call("sl_angle_table", out.data_ptr(), positions.data_ptr(), self._dev.data_ptr(), T, n, N.stream())
            return out
        ang = positions.to(torch.float64).unsqueeze(-1) * self._dev
        return torch.stack([ang.cos(), ang.sin()], -1).to(torch.float32)
