"""Zidalix: a decoder whose layers add attention over a compressed key/value latent and a clamped gated
feed-forward network, both reading the same residual stream.

This module is the configuration, the list of weights and a random initialisation; the serving model is
``rumus_b200/serve/zidalix.py``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch

from ..ops.rotary import RotarySpec
from ._weights import check_shapes, count


@dataclass(frozen=True)
class LatentAttentionConfig:
    """Per head ``dim`` unrotated and ``rot_dim`` rotated query / key dimensions and ``vdim`` value
    dimensions; keys and values are linear in a latent of ``kv_rank`` numbers per token.  ``kv_from``: the
    layer whose latents this one attends to instead of computing its own."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: RotarySpec
    kv_from: Optional[int] = None

    @staticmethod
    def from_dict(d: dict) -> "LatentAttentionConfig":
        m = LatentAttentionConfig(*(int(d[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank")),
                                  float(d["scale"]), RotarySpec.from_dict(d["rot"]),
                                  None if d.get("kv_from") is None else int(d["kv_from"]))
        if m.rot.dims != m.rot_dim or m.rot_dim % 2:
            raise ValueError(f"the rotated part of a head ({m.rot_dim}) must be even and equal rot.dims ({m.rot.dims})")
        return m


@dataclass(frozen=True)
class GatedMLPConfig:
    ff: int
    limit: float

    @staticmethod
    def from_dict(d: dict) -> "GatedMLPConfig":
        if d["kind"] != "dense":
            raise ValueError(f"unknown feed-forward kind {d['kind']!r}")
        return GatedMLPConfig(int(d["ff"]), float(d["limit"]))


@dataclass(frozen=True)
class ZidalixLayer:
    mixer: LatentAttentionConfig
    mlp: Optional[GatedMLPConfig]


@dataclass(frozen=True)
class ZidalixConfig:
    vocab_size: int
    d_model: int
    norm_eps: float
    embedding_scale: float
    logit_scale: float
    layers: Tuple[ZidalixLayer, ...]

    @staticmethod
    def from_dict(d: dict) -> "ZidalixConfig":
        layers: List[ZidalixLayer] = []
        for i, e in enumerate(d["layers"]):
            if e["type"] != "latent_attention":
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            mx = LatentAttentionConfig.from_dict(e["mixer"])
            if mx.kv_from is not None:
                j = mx.kv_from
                if not 0 <= j < i or layers[j].mixer.kv_from is not None:
                    raise ValueError(f"layer {i}: kv_from must name an earlier layer with latents of its own")
                o = layers[j].mixer
                if (o.kv_rank, o.rot_dim, o.rot) != (mx.kv_rank, mx.rot_dim, mx.rot):
                    raise ValueError(f"layer {i}: kv_rank, rot_dim and rotation differ from layer {j}'s")
            layers.append(ZidalixLayer(mx, None if e.get("mlp") is None else GatedMLPConfig.from_dict(e["mlp"])))
        return ZidalixConfig(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), float(d["embedding"]["scale"]),
                             float(d["logit_scale"]), tuple(layers))

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def weight_shapes(self) -> Dict[str, Tuple[int, ...]]:
        """Name -> shape of every checkpoint tensor (linear weights are ``[out, in]``)."""
        d = self.d_model
        s: Dict[str, Tuple[int, ...]] = {"embed": (self.vocab_size, d)}
        for i, L in enumerate(self.layers):
            m, p = L.mixer, f"l{i}."
            s[p + "norm1"] = (d,)
            s[p + "mix.q"] = (m.heads * (m.dim + m.rot_dim), d)
            if m.kv_from is None:
                s[p + "mix.dkv"] = (m.kv_rank + m.rot_dim, d)
                s[p + "mix.dkv.norm"] = (m.kv_rank,)
            s[p + "mix.uk"] = (m.heads * m.dim, m.kv_rank)
            s[p + "mix.uv"] = (m.heads * m.vdim, m.kv_rank)
            s[p + "mix.sink"] = (m.heads,)
            s[p + "mix.g"] = (m.heads * m.vdim, d)
            s[p + "mix.o"] = (d, m.heads * m.vdim)
            if L.mlp is not None:
                s[p + "norm2"] = (d,)
                s[p + "mlp.gate"] = (L.mlp.ff, d)
                s[p + "mlp.up"] = (L.mlp.ff, d)
                s[p + "mlp.down"] = (d, L.mlp.ff)
        s["final.norm"] = (d,)
        s["head"] = (self.vocab_size, d)
        return s

    def num_params(self) -> int:
        return count(self.weight_shapes())

    def check_weights(self, weights: Dict[str, torch.Tensor]) -> None:
        # a layer without a feed-forward has no use for its second norm; a checkpoint may carry it all the same
        check_shapes(weights, self.weight_shapes(), idle=[f"l{i}.norm2" for i, L in enumerate(self.layers) if L.mlp is None])

    def random_weights(self, seed: int = 0, device="cpu", dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
        """Normal weights of standard deviation 1/sqrt(in), norms of one, sinks of zero mean."""
        g = torch.Generator(device=device).manual_seed(seed)
        out = {}
        for k, shape in self.weight_shapes().items():
            if k.endswith("norm1") or k.endswith("norm2") or k.endswith(".norm"):
                out[k] = torch.ones(shape, dtype=dtype, device=device)
            else:
                std = 1.0 if k == "embed" or len(shape) == 1 else shape[1] ** -0.5
                out[k] = (torch.randn(shape, generator=g, device=device) * std).to(dtype)
        return out
