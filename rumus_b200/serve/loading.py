"""From a checkpoint folder (``config.json`` + ``model.safetensors``) to a running engine."""
from __future__ import annotations

import os

import torch

from ..io.safetensors import load_tensors
from ..models.registry import load_config
from .engine import Engine, ServeConfig


def load_engine(folder: str, device, dtype: torch.dtype = torch.bfloat16, **serve_kw) -> Engine:
    """The model class follows from the configuration's ``architecture``; ``serve_kw`` are fields of
    ``ServeConfig`` (pool size, block size, batch limits, ...)."""
    cfg = ServeConfig(model=load_config(folder), dtype=dtype, **serve_kw)
    return Engine(cfg, device, weights=load_tensors(os.path.join(folder, "model.safetensors")))
