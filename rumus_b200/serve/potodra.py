"""Potodra for the serving engine: weights in the layout the kernels take, and the decoder stack.

The model is a list of sub-layers (mixers and feed-forwards in turn).  The fp32 streams are read and written between
two of them only, by one kernel that mixes them, adds the last result and norms the next input; a sub-layer is a
function from that input to an fp32 result (and, for a mixture, rows of it that the kernel adds up).

* Everything a mixer projects from its input comes out of one matrix product, but for the few numbers per token that
  drive a recurrence, which stay in fp32.
* The two halves of a parallel mixer put their heads side by side, already scaled, and share the output product.
* Keys and values live in the paged cache, recurrent state in the sequence's slot (``HybridCache``).

What it shares with other decoders is in ``DecoderServing``.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..models.potodra import AttentionConfig, DenseConfig, MlstmConfig, ParallelConfig, PotodraConfig
from ..ops import moe, recurrent, stream, window
from ..ops.stream import pad8, pad_heads, pad_to
from .batch import StepBatch
from .cache import HybridCache
from .decoder import DecoderServing, Step, Weights

UNIT_SLOPE, UNIT_SHIFT = 1.702, 1.0      # gated units of experts: g sigmoid(1.702 g) (u + 1)


class PotodraServing(DecoderServing):
    name = "Potodra"

    def __init__(self, cfg, device, rank: int = 0, world: int = 1, seed: int = 0,
                 weights: Optional[Dict[str, torch.Tensor]] = None):
        super().__init__(cfg, device, seed, weights)
        m: PotodraConfig = cfg.model
        self.side = torch.cuda.Stream(self.device)   # the experts of a small batch run beside the shared one
        emb = self._get("embed")
        self.emb = emb.contiguous()
        self.head = pad_to(emb, m.vocab_size, self.dp).contiguous()
        self.subs: List[Weights] = []
        for i, L in enumerate(m.layers):
            load = {AttentionConfig: self._load_attention, MlstmConfig: self._load_mlstm, ParallelConfig: self._load_parallel}
            self._add(i, 1, load[type(L.mixer)](f"l{i}.mix.", L.mixer))
            if L.mlp is not None:
                self._add(i, 2, (self._load_dense if isinstance(L.mlp, DenseConfig) else self._load_mixture)(f"l{i}.mlp.", L.mlp))
        self.sum = torch.ones(m.streams, device=self.device)
        self.norm_f = self._f32("final.norm")
        self.attends = [s for s in self.subs if hasattr(s, "attention")]
        self.tiled_prompts = not self.exact and all(
            window.prefill_covered(cfg.dtype, s.dim_p, s.vdim_p, cfg.block_size, s.attention.scale) for s in self.attends)
        del self.weights

    @staticmethod
    def check_sizes(m: PotodraConfig) -> None:
        def most(i, what, n, limit):
            if n > limit:
                raise ValueError(f"layer {i}: {what} {n}, at most {limit}")

        if m.streams > stream.MAX_STREAMS:
            raise ValueError(f"{m.streams} streams, at most {stream.MAX_STREAMS}")
        for i, L in enumerate(m.layers):
            x = L.mixer
            for a in [x] if isinstance(x, AttentionConfig) else [x.left] if isinstance(x, ParallelConfig) else []:
                most(i, "numbers per attention head", max(a.dim, a.vdim), window.MAX_HEAD)
            for r in [x] if isinstance(x, MlstmConfig) else [x.right] if isinstance(x, ParallelConfig) else []:
                most(i, "key numbers per recurrent head", r.dim, recurrent.MAX_DIM)
            if L.mlp is not None and not isinstance(L.mlp, DenseConfig):
                most(i, "experts", L.mlp.experts, moe.MAX_EXPERTS)
                most(i, "groups of experts", L.mlp.groups, moe.MAX_GROUPS)

    # ------------------------------------------------------------------ weights
    def _add(self, layer: int, q: int, s: Weights) -> None:
        p = f"l{layer}."
        s.layer, s.norm = layer, self._f32(f"{p}norm{q}")
        s.hc_in, s.hc_out, s.hc_mix = (self._f32(f"{p}hc{q}.{k}") for k in ("in", "out", "mix"))
        self.subs.append(s)

    def _attention_rows(self, s: Weights, p: str, a: AttentionConfig, out_scale: float):
        """Fields of the attention part of a mixer; its input rows and biases [q | k | v]."""
        s.attention, s.out_scale = a, out_scale
        s.dim_p, s.vdim_p = pad8(a.dim), pad8(a.vdim)
        s.o_cols = a.heads * s.vdim_p
        s.sink = self._f32(p + "sink") if a.sink else None
        s.window = window.UNBOUNDED if a.window is None else a.window
        s.rot_id = self._rotation(a.rot) if a.rot.dims else -1
        parts = (("q", a.heads, a.dim), ("k", a.kv_heads, a.dim), ("v", a.kv_heads, a.vdim))
        return ([self._heads(p + k, n, size) for k, n, size in parts],
                [self._by_head(self._get(p + k + ".b"), n, size) for k, n, size in parts])

    def _load_attention(self, p: str, a: AttentionConfig) -> Weights:
        s = Weights()
        s.run = self._attention
        rows, bias = self._attention_rows(s, p, a, 1.0)
        s.w_in, s.b_in = torch.cat(rows).contiguous(), torch.cat(bias).contiguous()
        s.w_out = self._head_columns(p + "o", a.heads, a.vdim).contiguous()
        return s

    def _load_mlstm(self, p: str, c: MlstmConfig) -> Weights:
        s = Weights()
        s.run, s.mlstm = self._mlstm, c
        H, (d, e) = c.heads, (pad8(c.dim), pad8(c.vdim))
        s.w_in = torch.cat([self._heads(p + k, H, n) for k, n in (("q", c.dim), ("k", c.dim), ("v", c.vdim), ("g", c.vdim))]).contiguous()
        s.g_col, s.o_cols = H * (2 * d + e), H * e
        s.w_few = torch.cat([pad_to(self._get(p + k), H, self.dp) for k in ("i", "f")]).contiguous()
        s.b_few = torch.cat([self._get(p + k + ".b") for k in ("i", "f")]).contiguous()
        s.b_few32 = s.b_few.float()
        s.head_norm = self._by_head(self._f32(p + "norm"), H, c.vdim)
        s.w_out = self._head_columns(p + "o", H, c.vdim).contiguous()
        s.chunked = recurrent.mlstm_chunks_covered(self.cfg.dtype, d, e)
        s.state = {"S": ((H, d, e), torch.float32), "n": ((H, d), torch.float32), "m": ((H,), torch.float32)}
        return s

    def _load_parallel(self, p: str, c: ParallelConfig) -> Weights:
        s, r, left, right = Weights(), c.right, p + "left.", p + "right."
        s.run = self._parallel
        rows, bias = self._attention_rows(s, left, c.left, c.left_scale)
        H = r.heads
        s.raw_col = sum(x.shape[0] for x in rows)
        rows += self._delta_rows(s, right, r)
        s.head_norm = s.head_norm * c.right_scale
        s.low = []                                     # low-rank projections: first column, inner width, second factor
        for a, b, size in (("a1", "a2", r.dim), ("g1", "g2", r.vdim)):
            w1, w2 = self._get(right + a), self._get(right + b)
            inner = pad8(w1.shape[0])
            s.low.append((sum(x.shape[0] for x in rows), inner, pad_heads(w2, H, (size,), inner).contiguous()))
            rows.append(pad_to(w1, inner, self.dp))
        s.w_in = torch.cat(rows).contiguous()
        s.b_in = torch.cat(bias + [bias[0].new_zeros(s.w_in.shape[0] - s.raw_col)]).contiguous()
        s.w_few, s.b_few, s.b_few32 = pad_to(self._get(right + "b"), pad8(H), self.dp).contiguous(), None, None
        s.dt = self._by_head(self._f32(right + "dt_bias"), H, r.dim)
        s.w_out = torch.cat([self._head_columns(left + "o", c.left.heads, c.left.vdim), self._head_columns(right + "o", H, r.vdim)],
                            1).contiguous()
        return s

    def _load_dense(self, p: str, c: DenseConfig) -> Weights:
        s, ff = Weights(), pad8(c.ff)
        s.run = self._dense
        s.w_up = pad_to(self._get(p + "up"), ff, self.dp).contiguous()
        s.w_down = pad_to(self._get(p + "down"), self.model.d_model, ff).contiguous()
        return s

    def _load_mixture(self, p: str, c) -> Weights:
        s, dp, D = Weights(), self.dp, self.model.d_model
        s.run, s.mixture = self._mixture, c
        s.ff_p = pad8(c.shared_ff)
        # the last row's product gates the shared expert
        s.w_in = torch.cat([pad_to(self._get(p + "shared." + k), s.ff_p, dp) for k in ("gate", "up")]
                           + [pad_to(self._get(p + "shared.sg"), 8, dp)]).contiguous()
        s.w_down = pad_to(self._get(p + "shared.down"), D, s.ff_p).contiguous()
        s.router = pad_to(self._get(p + "router"), c.experts, dp).contiguous()
        s.correction = self._f32(p + "correction")

        def experts(name, *shape):
            return torch.stack([pad_to(self._get(f"{p}e{x}.{name}"), *shape) for x in range(c.experts)])

        s.w_gu = moe.interleave(experts("gate", c.ff, dp), experts("up", c.ff, dp))
        s.eff_p = s.w_gu.shape[1] // 2
        s.w_dn = experts("down", D, s.eff_p)
        s.counts = torch.zeros(c.experts + 1, dtype=torch.int32, device=self.device)
        return s

    # ------------------------------------------------------------------ what the engine calls
    def make_cache(self) -> HybridCache:
        c = self.cfg
        sizes, states = [None] * len(self.model.layers), [None] * len(self.model.layers)
        for s in self.subs:
            if hasattr(s, "attention"):
                sizes[s.layer] = (s.attention.kv_heads, s.dim_p, s.vdim_p)
            if hasattr(s, "state"):
                states[s.layer] = s.state
        return HybridCache(c.num_blocks, c.block_size, sizes, c.max_batch, states, c.dtype, self.device)

    def forward(self, batch: StepBatch, cache: HybridCache, row_parallel=None) -> torch.Tensor:
        """Hidden states ``[T, d]`` after the last layer and the final norm (activation type)."""
        m, dt, eps = self.model, self.cfg.dtype, self.model.norm_eps
        x = stream.embed_scaled(batch.tokens, self.emb, m.embedding_scale).unsqueeze(1).expand(-1, m.streams, -1)
        st = Step(batch, cache, [stream.rotary_table(batch.positions, f, s) for _, f, s in self.rotations])
        first = self.subs[0]
        h, x = stream.stream_mix_norm(x, first.hc_in, first.norm, eps, dt, self.dp)
        for i, s in enumerate(self.subs):
            y, rows = s.run(s, h, st)
            last = i + 1 == len(self.subs)
            w_in, norm = (self.sum, self.norm_f) if last else (self.subs[i + 1].hc_in, self.subs[i + 1].norm)
            h, x = stream.stream_mix_norm(x, w_in, norm, eps, dt, self.dp, y=y, mix=s.hc_mix, w_out=s.hc_out, add=rows, keep=not last)
        return h

    # ------------------------------------------------------------------ sub-layers: input -> (fp32 result, rows to add to it)
    def _attend(self, s: Weights, proj: torch.Tensor, out: torch.Tensor, st: Step) -> None:
        """Heads of every row into ``out``; this step's keys and values go to the cache first."""
        a, b = s.attention, st.batch
        k_pool, v_pool = st.cache.k[s.layer], st.cache.v[s.layer]
        rot = dict(tab=st.tabs[s.rot_id], rot=a.rot.dims, neighbours=a.neighbours) if s.rot_id >= 0 else {}
        window.window_post(proj, b.slots, k_pool, v_pool, a.heads, a.dim, **rot)
        q = proj[:, :a.heads * s.dim_p].unflatten(1, (a.heads, s.dim_p))
        more = dict(keep=a.keep_first, cap=a.softcap, out_scale=s.out_scale)
        if b.n_rows:
            n = b.n_rows
            window.window_rows_attention(q[:n], k_pool, v_pool, b.tables, b.ctx, s.sink, None, window.GATE_NONE, out[:n], s.window, a.scale,
                                         b.max_ctx, **more)
        if st.items is not None:
            window.window_prefill(q, k_pool, v_pool, b.seg_tables, st.items, s.sink, None, window.GATE_NONE, out, s.window, a.scale, **more)

    def _attention(self, s: Weights, h: torch.Tensor, st: Step):
        proj = self._mm(h, s.w_in, bias=s.b_in)
        out = self._heads_buffer(h, s.o_cols)
        self._attend(s, proj, out, st)
        return self._out(out, s.w_out), None

    def _mlstm(self, s: Weights, h: torch.Tensor, st: Step):
        c = s.mlstm
        gates, proj = self._few(s, h), self._mm(h, s.w_in)
        out = self._heads_buffer(h, s.o_cols)
        rest = (st.cache.state[s.layer], proj[:, s.g_col:], s.head_norm, out, c.dim, c.vdim, c.gate_cap, self.model.norm_eps)
        short, long = st.portions(s.chunked)
        recurrent.mlstm_rows(proj, gates, short, *rest)
        if long is not None:
            recurrent.mlstm_chunks(proj, gates, st.chunks(recurrent.MLSTM_CHUNK), long, *rest)
        return self._out(out, s.w_out), None

    def _parallel(self, s: Weights, h: torch.Tensor, st: Step):
        proj, few = self._mm(h, s.w_in, bias=s.b_in), self._few(s, h)
        out = self._heads_buffer(h, s.w_out.shape[1])
        self._attend(s, proj, out[:, :s.o_cols], st)
        (ac, an, a2), (gc, gn, g2) = s.low
        step, gate = self._out(proj[:, ac:ac + an], a2), self._mm(proj[:, gc:gc + gn], g2)
        self._delta(s, st, s.layer, proj[:, s.raw_col:], step, few, gate, out[:, s.o_cols:])
        return self._out(out, s.w_out), None

    def _dense(self, s: Weights, h: torch.Tensor, st: Step):
        return self._out(self._mm(h, s.w_up, act="relu2"), s.w_down), None

    def _mixture(self, s: Weights, h: torch.Tensor, st: Step):
        beside = h.shape[0] <= moe.ROUTE_ROWS
        if beside:
            self.side.wait_stream(torch.cuda.current_stream(self.device))
            with torch.cuda.stream(self.side):
                rows = self._experts(s, h)
        else:
            rows = self._experts(s, h)
        gu = self._mm(h, s.w_in)
        act = self._heads_buffer(h, s.ff_p)
        stream.clamped_glu(gu[:, :2 * s.ff_p], act, s.mixture.shared_limit, UNIT_SLOPE, UNIT_SHIFT, row_gate=gu[:, 2 * s.ff_p:])
        y = self._out(act, s.w_down)
        if beside:
            # what either stream allocated is used by the other between a fork and the join that follows it
            torch.cuda.current_stream(self.device).wait_stream(self.side)
        return y, rows

    def _experts(self, s: Weights, h: torch.Tensor):
        """Weighted outputs of the chosen experts, one row per (token, choice), and the rows of every token."""
        c, T = s.mixture, h.shape[0]
        logits = self._mm(h, s.router, out_dtype=torch.float32) if self.exact or T > moe.ROUTE_ROWS else None
        r = moe.route(h, s.router, s.correction, s.counts, c.top, logits=logits, plain=self.exact, score=moe.SIGMOID, groups=c.groups,
                      keep=c.keep)
        act = torch.empty((r.slots, s.eff_p), dtype=h.dtype, device=self.device)
        y = torch.empty((r.slots, self.dp), dtype=h.dtype, device=self.device)
        moe.grouped(h, s.w_gu, r, act, gated=True, plain=self.exact, unit=(c.limit, UNIT_SLOPE, UNIT_SHIFT))
        moe.grouped(act, s.w_dn, r, y, gated=False, plain=self.exact)
        return y, r.slot_of
