"""Potodra: a decoder whose residual is a few parallel streams (hyper-connections) and whose layers mix tokens in three
ways.

* "attention": grouped-query attention with biases, half-split rotation, soft-capped scores, a sink, and a sliding
  window that keeps the first tokens visible;
* "mlstm": a matrix memory per head with exponential input and forget gates;
* "parallel": plain causal attention (neighbour rotation) beside a gated delta rule with a decay per head and key
  channel, short convolutions and low-rank decay and gate projections; their results are added with fixed weights.

Feed-forwards are dense (squared relu) or mixtures of experts with group-limited sigmoid routing and a gated shared
expert.  Logits come from the embedding table.

This module is the configuration, the list of weights and a random initialisation; the serving model is
``rumus_b200/serve/potodra.py``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple, Union

import torch

from ..ops.rotary import RotarySpec
from ._weights import check_shapes, count


def _ints(d: dict, *keys: str):
    out = [int(d[k]) for k in keys]
    for k, n in zip(keys, out):
        if n < 1:
            raise ValueError(f"{k} = {n}")
    return out


@dataclass(frozen=True)
class AttentionConfig:
    """Query heads share key / value heads in groups.  ``window`` None: every earlier key is visible; else the last
    ``window`` keys and the sequence's first ``keep_first``.  ``softcap`` None: scores are not capped.
    ``neighbours``: rotation pairs elements 2i and 2i + 1, else i and i + dims / 2."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: RotarySpec
    neighbours: bool
    sink: bool
    window: Optional[int] = None
    keep_first: int = 0
    softcap: Optional[float] = None

    @staticmethod
    def from_dict(d: dict, neighbours: bool, sink: bool) -> "AttentionConfig":
        mask, cap = d.get("mask"), d.get("softcap")
        m = AttentionConfig(*_ints(d, "heads", "kv_heads", "dim", "vdim"), float(d["scale"]), RotarySpec.from_dict(d["rot"]),
                            neighbours, sink, _ints(mask, "size")[0] if mask else None,
                            int(mask.get("keep_first", 0)) if mask else 0, float(cap) if cap is not None else None)
        if m.heads % m.kv_heads:
            raise ValueError(f"{m.heads} query heads do not share {m.kv_heads} key/value heads evenly")
        if m.rot.dims % 2 or not 0 <= m.rot.dims <= m.dim:
            raise ValueError(f"rotation of {m.rot.dims} dimensions of a head of {m.dim}")
        if m.keep_first < 0 or (m.softcap is not None and not m.softcap > 0):
            raise ValueError(f"keep_first = {m.keep_first}, softcap = {m.softcap}")
        return m


@dataclass(frozen=True)
class MlstmConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @staticmethod
    def from_dict(d: dict) -> "MlstmConfig":
        return MlstmConfig(*_ints(d, "heads", "dim", "vdim"), float(d["gate_cap"]))


@dataclass(frozen=True)
class DeltaConfig:
    """Value heads share query / key heads in groups; ``conv``: taps of the short convolutions."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    @staticmethod
    def from_dict(d: dict) -> "DeltaConfig":
        m = DeltaConfig(*_ints(d, "heads", "kv_heads", "dim", "vdim", "conv"))
        if m.heads % m.kv_heads:
            raise ValueError(f"{m.heads} heads do not share {m.kv_heads} query/key heads evenly")
        return m


@dataclass(frozen=True)
class ParallelConfig:
    left: AttentionConfig
    right: DeltaConfig
    left_scale: float
    right_scale: float


Mixer = Union[AttentionConfig, MlstmConfig, ParallelConfig]


def mixer_from_dict(kind: str, d: dict) -> Mixer:
    if kind == "attention":
        return AttentionConfig.from_dict(d, neighbours=False, sink=True)
    if kind == "mlstm":
        return MlstmConfig.from_dict(d)
    if kind == "parallel":
        return ParallelConfig(AttentionConfig.from_dict(d["left"], neighbours=True, sink=False), DeltaConfig.from_dict(d["right"]),
                              float(d["left_scale"]), float(d["right_scale"]))
    raise ValueError(f"unknown mixer {kind!r}")


@dataclass(frozen=True)
class DenseConfig:
    ff: int


@dataclass(frozen=True)
class GroupedMixtureConfig:
    """Experts in ``groups`` equal groups of neighbours, of which the best ``keep`` are open to a token."""
    experts: int
    top: int
    groups: int
    keep: int
    ff: int
    limit: float
    shared_ff: int
    shared_limit: float


def mlp_from_dict(d: Optional[dict]) -> Union[DenseConfig, GroupedMixtureConfig, None]:
    if d is None:
        return None
    if d["kind"] == "dense":
        return DenseConfig(*_ints(d, "ff"))
    if d["kind"] != "moe":
        raise ValueError(f"unknown feed-forward kind {d['kind']!r}")
    r, e, s = d["router"], d["expert"], d["shared"]
    m = GroupedMixtureConfig(*_ints(r, "experts", "top"), *_ints(r["groups"], "count", "keep"), *_ints(e, "ff"), float(e["limit"]),
                             *_ints(s, "ff"), float(s["limit"]))
    if m.experts % m.groups or m.keep > m.groups or m.top > m.experts // m.groups * m.keep:
        raise ValueError(f"{m.top} of {m.experts} experts, {m.keep} of {m.groups} groups")
    return m


@dataclass(frozen=True)
class PotodraLayer:
    mixer: Mixer
    mlp: Union[DenseConfig, GroupedMixtureConfig, None]


@dataclass(frozen=True)
class PotodraConfig:
    vocab_size: int
    d_model: int
    norm_eps: float
    embedding_scale: float
    streams: int
    layers: Tuple[PotodraLayer, ...]

    @staticmethod
    def from_dict(d: dict) -> "PotodraConfig":
        layers: List[PotodraLayer] = []
        for i, e in enumerate(d["layers"]):
            try:
                layers.append(PotodraLayer(mixer_from_dict(e["type"], e["mixer"]), mlp_from_dict(e.get("mlp"))))
            except ValueError as err:
                raise ValueError(f"layer {i}: {err}") from None
        vocab, width, streams = _ints(d, "vocab", "width", "streams")
        return PotodraConfig(vocab, width, float(d["norm"]["eps"]), float(d["embedding"]["scale"]), streams, tuple(layers))

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def weight_shapes(self, ranks: Optional[Dict[int, Tuple[int, int]]] = None) -> Dict[str, Tuple[int, ...]]:
        """Name -> shape of every checkpoint tensor (linear weights are ``[out, in]``).  ``ranks``: inner widths of a
        layer's low-rank decay and gate projections, which only the tensors tell (default: the key size of a head)."""
        d, n = self.d_model, self.streams
        s: Dict[str, Tuple[int, ...]] = {"embed": (self.vocab_size, d)}

        def attention(p: str, m: AttentionConfig) -> None:
            for k, out in (("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
                s[p + k] = (out, d)
                s[p + k + ".b"] = (out,)
            if m.sink:
                s[p + "sink"] = (m.heads,)
            s[p + "o"] = (d, m.heads * m.vdim)

        def unit(p: str, ff: int) -> None:
            s[p + "gate"] = s[p + "up"] = (ff, d)
            s[p + "down"] = (d, ff)

        for i, L in enumerate(self.layers):
            p, m = f"l{i}.", L.mixer
            s[p + "norm1"] = (d,)
            if isinstance(m, AttentionConfig):
                attention(p + "mix.", m)
            elif isinstance(m, MlstmConfig):
                s[p + "mix.q"] = s[p + "mix.k"] = (m.heads * m.dim, d)
                s[p + "mix.v"] = s[p + "mix.g"] = (m.heads * m.vdim, d)
                s[p + "mix.o"], s[p + "mix.norm"] = (d, m.heads * m.vdim), (m.heads * m.vdim,)
                for k in ("i", "f"):
                    s[p + "mix." + k], s[p + "mix." + k + ".b"] = (m.heads, d), (m.heads,)
            else:
                attention(p + "mix.left.", m.left)
                r, o, e = m.right, p + "mix.right.", m.right.heads * m.right.vdim
                ra, rg = (ranks or {}).get(i, (r.dim, r.dim))
                for k, out in (("q", r.kv_heads * r.dim), ("k", r.kv_heads * r.dim), ("v", e)):
                    s[o + k], s[o + k + ".conv"] = (out, d), (out, r.conv)
                s[o + "b"], s[o + "A_log"], s[o + "norm"] = (r.heads, d), (r.heads,), (r.vdim,)
                s[o + "a1"], s[o + "a2"], s[o + "dt_bias"] = (ra, d), (r.heads * r.dim, ra), (r.heads * r.dim,)
                s[o + "g1"], s[o + "g2"], s[o + "o"] = (rg, d), (e, rg), (d, e)
            if isinstance(L.mlp, DenseConfig):
                s[p + "mlp.up"], s[p + "mlp.down"] = (L.mlp.ff, d), (d, L.mlp.ff)
            elif L.mlp is not None:
                for x in range(L.mlp.experts):
                    unit(f"{p}mlp.e{x}.", L.mlp.ff)
                s[p + "mlp.router"], s[p + "mlp.correction"] = (L.mlp.experts, d), (L.mlp.experts,)
                unit(p + "mlp.shared.", L.mlp.shared_ff)
                s[p + "mlp.shared.sg"] = (1, d)
            if L.mlp is not None:
                s[p + "norm2"] = (d,)
            for q in (1, 2) if L.mlp is not None else (1,):
                s[f"{p}hc{q}.in"] = s[f"{p}hc{q}.out"] = (n,)
                s[f"{p}hc{q}.mix"] = (n, n)
        s["final.norm"] = (d,)
        return s

    def ranks_of(self, weights: Dict[str, torch.Tensor]) -> Dict[int, Tuple[int, int]]:
        out = {}
        for i, L in enumerate(self.layers):
            a, g = (weights.get(f"l{i}.mix.right.{k}") for k in ("a1", "g1"))
            if isinstance(L.mixer, ParallelConfig) and a is not None and g is not None:
                out[i] = (a.shape[0], g.shape[0])
        return out

    def num_params(self) -> int:
        return count(self.weight_shapes())

    def check_weights(self, weights: Dict[str, torch.Tensor]) -> None:
        # a layer without a feed-forward may still carry the norm and connections of one
        idle = [f"l{i}.{k}" for i, L in enumerate(self.layers) if L.mlp is None for k in ("norm2", "hc2.in", "hc2.out", "hc2.mix")]
        check_shapes(weights, self.weight_shapes(self.ranks_of(weights)), idle)

    def random_weights(self, seed: int = 0, device="cpu", dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
        """Normal weights of standard deviation 1/sqrt(in); norms of one; streams that keep to themselves and share
        their mean; forget gates that mostly remember, slow decays."""
        g = torch.Generator(device=device).manual_seed(seed)
        out = {}
        for k, shape in self.weight_shapes().items():
            last = k.rsplit(".", 1)[-1]
            if last in ("norm", "norm1", "norm2"):
                t = torch.ones(shape, device=device)
            elif last == "in":
                t = torch.full(shape, 1.0 / self.streams, device=device)
            elif last == "out":
                t = torch.ones(shape, device=device)
            elif last == "mix":
                t = torch.eye(self.streams, device=device)
            elif last == "A_log":
                t = torch.zeros(shape, device=device)
            elif last == "dt_bias":
                t = torch.full(shape, -4.0, device=device)
            elif k.endswith(".f.b"):
                t = torch.full(shape, 4.0, device=device)
            elif len(shape) == 1:
                t = 0.1 * torch.randn(shape, generator=g, device=device)
            else:
                t = torch.randn(shape, generator=g, device=device) * (1.0 if k == "embed" else shape[1] ** -0.5)
            out[k] = t.to(dtype)
        return out
