"""Lerosun for the serving engine: weights in the layout the kernels take, and the decoder stack.

The model is a list of sub-layers (mixers and feed-forwards in turn) in the order they run; the passes of a loop share
the sub-layers' weights, and a run has its own number for the cache.  The fp32 residual is read and written between two
sub-layers only, by one kernel that adds the last result, scaled channel by channel, and norms the next input.

* Everything a mixer projects from its input comes out of one matrix product, but for the two numbers per token and head
  that drive a delta rule, which stay in fp32.
* Values are never projected: the kernel that rotates the keys puts them into the cache in both forms.
* Keys and values live in the paged cache, recurrent state in the sequence's slot (``HybridCache``).
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..models.lerosun import LerosunConfig, TalkingAttentionConfig
from ..ops import recurrent, stream, talk, window
from ..ops.stream import pad8, pad_to
from .batch import StepBatch
from .cache import HybridCache
from .decoder import DecoderServing, Step, Weights


class LerosunServing(DecoderServing):
    name = "Lerosun"

    def __init__(self, cfg, device, rank: int = 0, world: int = 1, seed: int = 0,
                 weights: Optional[Dict[str, torch.Tensor]] = None):
        super().__init__(cfg, device, seed, weights)
        m: LerosunConfig = cfg.model
        self.emb = self._get("embed").contiguous()
        self.head = pad_to(self._get("head"), m.vocab_size, self.dp).contiguous()
        self.norm_e, self.norm_f = self._one("embed.norm"), self._one("final.norm")
        self.mixers: List[Weights] = []
        by_layer: List[List[Weights]] = []
        for i, L in enumerate(m.layers):
            load = self._load_attention if isinstance(L.mixer, TalkingAttentionConfig) else self._load_delta
            parts = [load(f"l{i}.mix.", L.mixer)]
            if L.mlp is not None:
                parts.append(self._load_dense(f"l{i}.mlp.", L.mlp))
            for q, s in enumerate(parts, 1):
                s.norm, s.scale = self._one(f"l{i}.norm{q}"), self._f32(f"l{i}.ls{q}")
            self.mixers.append(parts[0])
            by_layer.append(parts)
        self.runs = [(s, run) for run, i in enumerate(m.runs) for s in by_layer[i]]      # (sub-layer, number of its layer's run)
        self.tiled_prompts = not self.exact and all(
            talk.prefill_covered(cfg.dtype, s.attention.heads, s.attention.kv_heads, s.dim_p, s.dim_p, cfg.block_size, s.attention.scale)
            for s in self.mixers if hasattr(s, "attention"))
        del self.weights

    @staticmethod
    def check_sizes(m: LerosunConfig) -> None:
        for i, L in enumerate(m.layers):
            x = L.mixer
            if isinstance(x, TalkingAttentionConfig):
                if not talk.rows_covered(x.heads, pad8(x.dim), pad8(x.dim)):
                    raise ValueError(f"layer {i}: {x.heads} talking heads of {x.dim} numbers do not fit a CTA's shared memory")
            elif x.dim > recurrent.MAX_DIM:
                raise ValueError(f"layer {i}: key numbers per recurrent head {x.dim}, at most {recurrent.MAX_DIM}")

    # ------------------------------------------------------------------ weights
    def _one(self, name: str) -> torch.Tensor:
        return self._f32(name).view(1)

    def _load_attention(self, p: str, a: TalkingAttentionConfig) -> Weights:
        s = Weights()
        s.run, s.attention, s.dim_p = self._attention, a, pad8(a.dim)
        rows = [self._heads(p + "q", a.heads, a.dim), self._heads(p + "k", a.kv_heads, a.dim)]
        bias = [self._by_head(self._get(p + k + ".b"), n, a.dim) for k, n in (("q", a.heads), ("k", a.kv_heads))]
        s.g_col = sum(x.shape[0] for x in rows)
        rows.append(pad_to(self._get(p + "g"), pad8(a.heads), self.dp))
        s.w_in, s.b_in = torch.cat(rows).contiguous(), torch.cat(bias + [bias[0].new_zeros(pad8(a.heads))]).contiguous()
        s.mix = (self._f32(p + "talk") * self._f32(p + "temp")).contiguous()      # a temperature per listened-to head
        s.sink = self._f32(p + "sink")
        s.rot_id = self._rotation(a.rot) if a.rot.dims else -1
        s.w_out = self._head_columns(p + "o", a.heads, a.dim).contiguous()
        return s

    def _load_delta(self, p: str, r) -> Weights:
        s = Weights()
        s.run = self._delta_rule
        rows = self._delta_rows(s, p, r)
        s.g_col = sum(x.shape[0] for x in rows)
        s.w_in = torch.cat(rows + [self._heads(p + "g", r.heads, r.vdim)]).contiguous()
        s.o_cols, s.few = r.heads * pad8(r.vdim), pad8(r.heads)
        s.w_few = torch.cat([pad_to(self._get(p + k), s.few, self.dp) for k in ("b", "a")]).contiguous()
        s.b_few = s.b_few32 = None
        s.dt = self._f32(p + "dt_bias")
        s.w_out = self._head_columns(p + "o", r.heads, r.vdim).contiguous()
        return s

    def _load_dense(self, p: str, c) -> Weights:
        s = Weights()
        s.run, s.ff_p = self._dense, pad8(c.ff)
        s.w_in = torch.cat([pad_to(self._get(p + k), s.ff_p, self.dp) for k in ("gate", "up")]).contiguous()
        s.w_down = pad_to(self._get(p + "down"), self.model.d_model, s.ff_p).contiguous()
        return s

    # ------------------------------------------------------------------ what the engine calls
    def make_cache(self) -> HybridCache:
        c, mixers = self.cfg, [self.mixers[i] for i in self.model.runs]
        sizes = [(s.attention.kv_heads, s.dim_p, s.dim_p) if hasattr(s, "attention") else None for s in mixers]
        return HybridCache(c.num_blocks, c.block_size, sizes, c.max_batch, [getattr(s, "state", None) for s in mixers], c.dtype, self.device)

    def forward(self, batch: StepBatch, cache: HybridCache, row_parallel=None) -> torch.Tensor:
        """Hidden states ``[T, d]`` after the last layer and the final norm (activation type)."""
        dt, eps = self.cfg.dtype, self.model.norm_eps
        st = Step(batch, cache, [stream.rotary_table(batch.positions, f, s) for _, f, s in self.rotations])
        norms = [s.norm for s, _ in self.runs] + [self.norm_f]
        x, h = stream.embed_norm(batch.tokens, self.emb, self.norm_e, norms[0], eps, self.dp)
        for i, (s, run) in enumerate(self.runs):
            y = s.run(s, run, h, st)
            h = stream.scaled_add_norm(x, y, s.scale, norms[i + 1], eps, dt, self.dp, keep=i + 1 < len(self.runs))
        return h

    # ------------------------------------------------------------------ sub-layers: input -> fp32 result
    def _attention(self, s: Weights, run: int, h: torch.Tensor, st: Step) -> torch.Tensor:
        a, b, k_pool, v_pool = s.attention, st.batch, st.cache.k[run], st.cache.v[run]
        proj = self._mm(h, s.w_in, bias=s.b_in)
        rot = dict(tab=st.tabs[s.rot_id], rot=a.rot.dims) if s.rot_id >= 0 else {}
        n, gate, out = b.n_rows, proj[:, s.g_col:], self._heads_buffer(h, a.heads * s.dim_p)
        qmix = talk.talk_post(proj, b.slots, k_pool, v_pool, s.mix, a.heads, n, **rot)
        if n:
            q = proj[:n, :a.heads * s.dim_p].unflatten(1, (a.heads, s.dim_p))
            talk.talk_rows_attention(q, k_pool, v_pool, b.tables, b.ctx, s.mix, s.sink, gate[:n], window.GATE_HEAD, out[:n], a.window, a.scale,
                                     b.max_ctx)
        if st.items is not None:
            talk.talk_prefill(qmix, n, k_pool, v_pool, b.seg_tables, st.items, s.sink, gate, window.GATE_HEAD, out, a.window, a.scale)
        return self._out(out, s.w_out)

    def _delta_rule(self, s: Weights, run: int, h: torch.Tensor, st: Step) -> torch.Tensor:
        few, proj = self._few(s, h), self._mm(h, s.w_in)
        out = self._heads_buffer(h, s.o_cols)
        self._delta(s, st, run, proj, few[:, s.few:], few, proj[:, s.g_col:], out, per_head=True, silu=True)
        return self._out(out, s.w_out)

    def _dense(self, s: Weights, run: int, h: torch.Tensor, st: Step) -> torch.Tensor:
        act = self._heads_buffer(h, s.ff_p)
        stream.glu(stream.GLU_RELU, self._mm(h, s.w_in), act)
        return self._out(act, s.w_down)
