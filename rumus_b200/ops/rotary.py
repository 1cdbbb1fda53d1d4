"""Rotary frequencies: plain, and YaRN's blend of interpolated and unchanged frequencies.

The kernels take a per-step table of (cos, sin) rows, so a new frequency rule is a new function here.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional, Tuple

import torch


@dataclass(frozen=True)
class YarnScaling:
    factor: float
    original: float      # context length the unscaled model was made for
    fast: float          # pairs that turn more often than this over `original` tokens keep their frequency
    slow: float          # pairs that turn less often than this are divided by `factor`


@dataclass(frozen=True)
class RotarySpec:
    """``dims`` rotated dimensions, neighbouring elements (2i, 2i+1) forming pair i."""
    base: float
    dims: int
    scaling: Optional[YarnScaling] = None

    @staticmethod
    def from_dict(d: dict) -> "RotarySpec":
        s = d.get("scaling")
        return RotarySpec(float(d["base"]), int(d["dims"]),
                          None if s is None else YarnScaling(*(float(s[k]) for k in ("factor", "original", "fast", "slow"))))

    def frequencies(self) -> Tuple[torch.Tensor, float]:
        """(frequency of every pair, factor on cos and sin)."""
        dims, base, sc = self.dims, self.base, self.scaling
        i = torch.arange(dims // 2, dtype=torch.float64)
        f = base ** (-2.0 * i / dims)
        if sc is None:
            return f.float(), 1.0

        def index(turns: float) -> float:      # pair index (as a dimension) that turns `turns` times
            return dims * math.log(sc.original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

        lo = max(math.floor(index(sc.fast)), 0)
        hi = min(math.ceil(index(sc.slow)), dims - 1)
        ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        return (f / sc.factor * ramp + f * (1.0 - ramp)).float(), 0.1 * math.log(sc.factor) + 1.0
