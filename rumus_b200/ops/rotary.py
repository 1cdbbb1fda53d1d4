"""Rotary frequencies: plain, YaRN's blend by pair index, and a blend by wavelength (as in Llama 3.1).

The kernels take a per-step table of (cos, sin) rows, so a new frequency rule is a new scaling class here.
Which two elements of a head form pair i is the kernel's affair (neighbours in ``latent_post``, halves in
``window_post``).
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional, Tuple, Union

import torch


@dataclass(frozen=True)
class YarnScaling:
    factor: float
    original: float      # context length the unscaled model was made for
    fast: float          # pairs that turn more often than this over `original` tokens keep their frequency
    slow: float          # pairs that turn less often than this are divided by `factor`

    def apply(self, f: torch.Tensor, base: float, dims: int) -> Tuple[torch.Tensor, float]:
        def index(turns: float) -> float:      # pair index (as a dimension) that turns `turns` times
            return dims * math.log(self.original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

        lo = max(math.floor(index(self.fast)), 0)
        hi = min(math.ceil(index(self.slow)), dims - 1)
        i = torch.arange(dims // 2, dtype=torch.float64)
        ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        return f / self.factor * ramp + f * (1.0 - ramp), 0.1 * math.log(self.factor) + 1.0


@dataclass(frozen=True)
class BandScaling:
    """Blend by the number of turns over ``original`` tokens: ``high`` or more keep their frequency, ``low`` or
    fewer are divided by ``factor``, linear in the turns between."""
    factor: float
    low: float
    high: float
    original: float

    def apply(self, f: torch.Tensor, base: float, dims: int) -> Tuple[torch.Tensor, float]:
        wave = 2.0 * math.pi / f
        s = (self.original / wave - self.low) / (self.high - self.low) if self.high != self.low else torch.zeros_like(f)
        out = (1.0 - s) * f / self.factor + s * f
        out = torch.where(wave > self.original / self.low, f / self.factor, out)
        return torch.where(wave < self.original / self.high, f, out), 1.0


Scaling = Union[YarnScaling, BandScaling]


def scaling_from_dict(d: Optional[dict]) -> Optional[Scaling]:
    """The rule follows from the keys."""
    if d is None:
        return None
    for cls, keys in ((YarnScaling, ("factor", "original", "fast", "slow")), (BandScaling, ("factor", "low", "high", "original"))):
        if set(keys) <= set(d):
            return cls(*(float(d[k]) for k in keys))
    raise ValueError(f"unknown frequency scaling with keys {sorted(d)}")


@dataclass(frozen=True)
class RotarySpec:
    """``dims`` rotated dimensions of a head: pair i turns by position x base^(-2i/dims), scaled."""
    base: float
    dims: int
    scaling: Optional[Scaling] = None

    @staticmethod
    def from_dict(d: dict) -> "RotarySpec":
        return RotarySpec(float(d["base"]), int(d["dims"]), scaling_from_dict(d.get("scaling")))

    def frequencies(self) -> Tuple[torch.Tensor, float]:
        """(frequency of every pair, factor on cos and sin)."""
        f = self.base ** (-2.0 * torch.arange(self.dims // 2, dtype=torch.float64) / self.dims)
        if self.scaling is None:
            return f.float(), 1.0
        f, factor = self.scaling.apply(f, self.base, self.dims)
        return f.float(), factor
