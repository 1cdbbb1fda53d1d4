"""Lerosun: a decoder of gated delta rules and sliding-window attention whose heads talk.

* "delta": a gated delta rule with one decay per head, short convolutions, and a silu output gate;
* "attention": grouped-query attention over a sliding window; keys are rotated, values are the same keys before their
  rotation; a head's scores have a temperature and are mixed with the other heads' before a softmax with a sink; one output
  gate per head.

Norms have one number for all channels, every sub-layer's result a weight per channel.  Feed-forwards are gated (relu).
Embeddings are normed.  A run of layers may be passed several times with the same weights; every pass has a cache or state
of its own.

This module is the configuration, the list of weights and a random initialisation; the serving model is
``rumus_b200/serve/lerosun.py``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple, Union

import torch

from ..ops.rotary import RotarySpec
from ._weights import check_shapes, count
from .potodra import DeltaConfig, DenseConfig, _ints


@dataclass(frozen=True)
class TalkingAttentionConfig:
    """Query heads share key / value heads in groups; a position sees itself and the ``window - 1`` before it.  Values are
    unrotated keys, so they have the keys' size."""
    heads: int
    kv_heads: int
    dim: int
    window: int
    scale: float
    rot: RotarySpec

    @staticmethod
    def from_dict(d: dict) -> "TalkingAttentionConfig":
        m = TalkingAttentionConfig(*_ints(d, "heads", "kv_heads", "dim"), *_ints(d["mask"], "size"), float(d["scale"]),
                                   RotarySpec.from_dict(d["rot"]))
        if m.heads % m.kv_heads:
            raise ValueError(f"{m.heads} query heads do not share {m.kv_heads} key/value heads evenly")
        if int(d.get("vdim", m.dim)) != m.dim:
            raise ValueError(f"values are keys, but have {d['vdim']} numbers and not {m.dim}")
        if m.rot.dims % 2 or not 0 <= m.rot.dims <= m.dim:
            raise ValueError(f"rotation of {m.rot.dims} dimensions of a head of {m.dim}")
        return m


Mixer = Union[TalkingAttentionConfig, DeltaConfig]


def mixer_from_dict(kind: str, d: dict) -> Mixer:
    if kind == "attention":
        return TalkingAttentionConfig.from_dict(d)
    if kind == "delta":
        return DeltaConfig.from_dict(d)
    raise ValueError(f"unknown mixer {kind!r}")


def mlp_from_dict(d: Optional[dict]) -> Optional[DenseConfig]:
    if d is None:
        return None
    if d["kind"] != "dense":
        raise ValueError(f"unknown feed-forward kind {d['kind']!r}")
    return DenseConfig(*_ints(d, "ff"))


@dataclass(frozen=True)
class LerosunLayer:
    mixer: Mixer
    mlp: Optional[DenseConfig]


@dataclass(frozen=True)
class LerosunConfig:
    vocab_size: int
    d_model: int
    norm_eps: float
    layers: Tuple[LerosunLayer, ...]
    loop: Tuple[int, int, int] = (0, 0, 1)       # first layer, one past the last, passes

    @staticmethod
    def from_dict(d: dict) -> "LerosunConfig":
        layers: List[LerosunLayer] = []
        for i, e in enumerate(d["layers"]):
            try:
                layers.append(LerosunLayer(mixer_from_dict(e["type"], e["mixer"]), mlp_from_dict(e.get("mlp"))))
            except ValueError as err:
                raise ValueError(f"layer {i}: {err}") from None
        lp = d.get("loop") or {"start": 0, "stop": 0, "times": 1}
        start, stop, times = (int(lp[k]) for k in ("start", "stop", "times"))
        if not 0 <= start <= stop <= len(layers) or times < 1:
            raise ValueError(f"a loop of {times} passes over layers {start} .. {stop} of {len(layers)}")
        return LerosunConfig(*_ints(d, "vocab", "width"), float(d["norm"]["eps"]), tuple(layers), (start, stop, times))

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def runs(self) -> List[int]:
        """Layer numbers in the order they run."""
        start, stop, times = self.loop
        return [*range(start), *list(range(start, stop)) * times, *range(stop, len(self.layers))]

    def weight_shapes(self) -> Dict[str, Tuple[int, ...]]:
        """Name -> shape of every checkpoint tensor (linear weights are ``[out, in]``)."""
        d = self.d_model
        s: Dict[str, Tuple[int, ...]] = {"embed": (self.vocab_size, d), "embed.norm": ()}
        for i, L in enumerate(self.layers):
            p, m = f"l{i}.", L.mixer
            o = p + "mix."
            s[p + "norm1"], s[p + "ls1"] = (), (d,)
            if isinstance(m, TalkingAttentionConfig):
                for k, n in (("q", m.heads), ("k", m.kv_heads)):
                    s[o + k], s[o + k + ".b"] = (n * m.dim, d), (n * m.dim,)
                s[o + "talk"], s[o + "temp"], s[o + "sink"] = (m.heads, m.heads), (m.heads,), (m.heads,)
                s[o + "g"], s[o + "o"] = (m.heads, d), (d, m.heads * m.dim)
            else:
                e = m.heads * m.vdim
                for k, out in (("q", m.kv_heads * m.dim), ("k", m.kv_heads * m.dim), ("v", e)):
                    s[o + k], s[o + k + ".conv"] = (out, d), (out, m.conv)
                s[o + "a"] = s[o + "b"] = (m.heads, d)
                s[o + "A_log"] = s[o + "dt_bias"] = (m.heads,)
                s[o + "norm"], s[o + "g"], s[o + "o"] = (m.vdim,), (e, d), (d, e)
            if L.mlp is not None:
                s[p + "norm2"], s[p + "ls2"] = (), (d,)
                s[p + "mlp.gate"] = s[p + "mlp.up"] = (L.mlp.ff, d)
                s[p + "mlp.down"] = (d, L.mlp.ff)
        s["final.norm"] = ()
        s["head"] = (self.vocab_size, d)
        return s

    def num_params(self) -> int:
        return count(self.weight_shapes())

    def check_weights(self, weights: Dict[str, torch.Tensor]) -> None:
        # a layer without a feed-forward may still carry the norm and weights of one
        idle = [f"l{i}.{k}" for i, L in enumerate(self.layers) if L.mlp is None for k in ("norm2", "ls2")]
        check_shapes(weights, self.weight_shapes(), idle)

    def random_weights(self, seed: int = 0, device="cpu", dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
        """Normal weights of standard deviation 1/sqrt(in); norms, temperatures and layer scales of one; heads that mostly
        listen to themselves; slow decays."""
        g = torch.Generator(device=device).manual_seed(seed)
        out = {}
        for k, shape in self.weight_shapes().items():
            last = k.rsplit(".", 1)[-1]
            if last in ("norm", "norm1", "norm2", "ls1", "ls2", "temp"):
                t = torch.ones(shape, device=device)
            elif last == "A_log":
                t = torch.zeros(shape, device=device)
            elif last == "dt_bias":
                t = torch.full(shape, -4.0, device=device)
            elif last == "talk":
                t = torch.eye(shape[0], device=device) + 0.5 / shape[0] * torch.randn(shape, generator=g, device=device)
            elif len(shape) == 1:
                t = 0.1 * torch.randn(shape, generator=g, device=device)
            else:
                t = torch.randn(shape, generator=g, device=device) * (1.0 if k == "embed" else shape[1] ** -0.5)
            out[k] = t.to(dtype)
        return out
