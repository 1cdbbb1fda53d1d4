"""Nufupel: a decoder whose layers add sliding-window attention and a feed-forward network that both read one
norm of the residual stream.

Two kinds of attention ("attention": no positions in the scores, an output gate per number; "attention_2":
query / key norm, rotation, an output gate per head), dense feed-forward layers and mixtures of experts with a
shared expert.  A layer may use an earlier layer's weights with a cache of its own.

This module is the configuration, the list of weights and a random initialisation; the serving model is
``rumus_b200/serve/nufupel.py``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple, Union

import torch

from ..ops.rotary import RotarySpec
from ._weights import check_shapes, count


@dataclass(frozen=True)
class WindowAttentionConfig:
    """Query heads share key / value heads in groups; a position sees itself and the ``window - 1`` before it.
    ``rot``: rotation of the first ``rot.dims`` dimensions, which comes with query / key norms and one output
    gate per head; None: neither, and one output gate per number."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    window: int
    scale: float
    rot: Optional[RotarySpec] = None

    @staticmethod
    def from_dict(kind: str, d: dict) -> "WindowAttentionConfig":
        if kind not in ("attention", "attention_2"):
            raise ValueError(f"unknown mixer {kind!r}")
        m = WindowAttentionConfig(*(int(d[k]) for k in ("heads", "kv_heads", "dim", "vdim")), int(d["mask"]["size"]),
                                  float(d["scale"]), RotarySpec.from_dict(d["rot"]) if kind == "attention_2" else None)
        if m.heads % m.kv_heads:
            raise ValueError(f"{m.heads} query heads do not share {m.kv_heads} key/value heads evenly")
        if m.window < 1:
            raise ValueError(f"a window of {m.window} tokens")
        if m.rot is not None and (m.rot.dims % 2 or m.rot.dims > m.dim):
            raise ValueError(f"{m.rot.dims} rotated dimensions of {m.dim}")
        return m

    @property
    def qk_norm(self) -> bool:
        return self.rot is not None

    @property
    def gate_per_head(self) -> bool:
        return self.rot is not None


@dataclass(frozen=True)
class DenseConfig:
    ff: int


@dataclass(frozen=True)
class MixtureConfig:
    experts: int
    top: int
    ff: int
    shared_ff: int


def mlp_from_dict(d: Optional[dict]) -> Union[DenseConfig, MixtureConfig, None]:
    if d is None:
        return None
    if d["kind"] == "dense":
        return DenseConfig(int(d["ff"]))
    if d["kind"] != "moe":
        raise ValueError(f"unknown feed-forward kind {d['kind']!r}")
    m = MixtureConfig(int(d["router"]["experts"]), int(d["router"]["top"]), int(d["expert"]["ff"]), int(d["shared"]["ff"]))
    if not 1 <= m.top <= m.experts:
        raise ValueError(f"{m.top} of {m.experts} experts")
    return m


@dataclass(frozen=True)
class NufupelLayer:
    mixer: WindowAttentionConfig
    mlp: Union[DenseConfig, MixtureConfig, None]
    owner: int                     # the layer whose weights this one uses (its own index: it has weights itself)


@dataclass(frozen=True)
class NufupelConfig:
    vocab_size: int
    d_model: int
    norm_eps: float
    embedding_scale: float
    logit_softcap: float
    layers: Tuple[NufupelLayer, ...]

    @staticmethod
    def from_dict(d: dict) -> "NufupelConfig":
        layers: List[NufupelLayer] = []
        for i, e in enumerate(d["layers"]):
            try:
                mx, mlp = WindowAttentionConfig.from_dict(e["type"], e["mixer"]), mlp_from_dict(e.get("mlp"))
            except ValueError as err:
                raise ValueError(f"layer {i}: {err}") from None
            owner, j = i, e.get("weights_of")
            if j is not None:
                if not 0 <= int(j) < len(d["layers"]) or int(j) == i or d["layers"][int(j)].get("weights_of") is not None:
                    raise ValueError(f"layer {i}: weights_of must name a layer with weights of its own")
                owner = int(j)
            layers.append(NufupelLayer(mx, mlp, owner))
        for i, L in enumerate(layers):
            o = layers[L.owner]
            if (o.mixer, o.mlp) != (L.mixer, L.mlp):
                raise ValueError(f"layer {i} differs from layer {L.owner}, whose weights it uses")
        return NufupelConfig(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), float(d["embedding"]["scale"]),
                             float(d["logit_softcap"]), tuple(layers))

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def weight_shapes(self) -> Dict[str, Tuple[int, ...]]:
        """Name -> shape of every checkpoint tensor (linear weights are ``[out, in]``)."""
        d = self.d_model
        s: Dict[str, Tuple[int, ...]] = {"embed": (self.vocab_size, d)}
        for i, L in enumerate(self.layers):
            if L.owner != i:
                continue
            m, p = L.mixer, f"l{i}."
            s[p + "norm1"] = (d,)
            s[p + "mix.q"] = (m.heads * m.dim, d)
            s[p + "mix.k"] = (m.kv_heads * m.dim, d)
            s[p + "mix.v"] = (m.kv_heads * m.vdim, d)
            if m.qk_norm:
                s[p + "mix.q.norm"] = s[p + "mix.k.norm"] = (m.dim,)
            s[p + "mix.sink"] = (m.heads,)
            s[p + "mix.g"] = (m.heads if m.gate_per_head else m.heads * m.vdim, d)
            s[p + "mix.o"] = (d, m.heads * m.vdim)

            def unit(name: str, ff: int) -> None:
                s[name + "gate"] = s[name + "up"] = (ff, d)
                s[name + "down"] = (d, ff)

            if isinstance(L.mlp, DenseConfig):
                unit(p + "mlp.", L.mlp.ff)
            elif L.mlp is not None:
                for e in range(L.mlp.experts):
                    unit(f"{p}mlp.e{e}.", L.mlp.ff)
                s[p + "mlp.router"] = (L.mlp.experts, d)
                s[p + "mlp.router.b"] = (L.mlp.experts,)
                unit(p + "mlp.shared.", L.mlp.shared_ff)
        s["final.norm"] = (d,)
        s["head"] = (self.vocab_size, d)
        return s

    def num_params(self) -> int:
        return count(self.weight_shapes())

    def check_weights(self, weights: Dict[str, torch.Tensor]) -> None:
        check_shapes(weights, self.weight_shapes())

    def random_weights(self, seed: int = 0, device="cpu", dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
        """Normal weights of standard deviation 1/sqrt(in); norms of one (the layers' and the final one are stored
        around zero), sinks and router biases of zero mean."""
        g = torch.Generator(device=device).manual_seed(seed)
        out = {}
        for k, shape in self.weight_shapes().items():
            if k.endswith("norm1") or k == "final.norm":
                out[k] = torch.zeros(shape, dtype=dtype, device=device)
            elif k.endswith(".norm"):
                out[k] = torch.ones(shape, dtype=dtype, device=device)
            else:
                std = 1.0 if k == "embed" or len(shape) == 1 else shape[1] ** -0.5
                out[k] = (torch.randn(shape, generator=g, device=device) * std).to(dtype)
        return out
