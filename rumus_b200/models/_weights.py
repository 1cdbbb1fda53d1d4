"""Checks of a checkpoint against the weights a configuration lists (name -> shape)."""
from __future__ import annotations

import math
from typing import Dict, Iterable, Tuple

import torch


def count(shapes: Dict[str, Tuple[int, ...]]) -> int:
    return sum(math.prod(s) for s in shapes.values())


def check_shapes(weights: Dict[str, torch.Tensor], want: Dict[str, Tuple[int, ...]], idle: Iterable[str] = ()) -> None:
    """``idle``: names a checkpoint may carry although the configuration has no use for them."""
    names = set(weights) - set(idle)
    missing, extra = sorted(set(want) - names), sorted(names - set(want))
    if missing or extra:
        raise ValueError(f"checkpoint does not fit the configuration: missing {missing[:5]}, unexpected {extra[:5]}")
    for k, shape in want.items():
        if tuple(weights[k].shape) != shape:
            raise ValueError(f"{k}: checkpoint shape {tuple(weights[k].shape)}, configuration {shape}")
