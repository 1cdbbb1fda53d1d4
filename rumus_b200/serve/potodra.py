"""Potodra for the serving engine: weights in the layout the kernels take, and the decoder stack.

The model is a list of sub-layers (mixers and feed-forwards in turn).  The fp32 streams are read and written between
two of them only, by one kernel that mixes them, adds the last result and norms the next input; a sub-layer is a
function from that input to an fp32 result (and, for a mixture, rows of it that the kernel adds up).

* Everything a mixer projects from its input comes out of one matrix product, but for the few numbers per token that
  drive a recurrence, which stay in fp32.
* The two halves of a parallel mixer put their heads side by side, already scaled, and share the output product.
* Keys and values live in the paged cache, recurrent state in the sequence's slot (``HybridCache``).

Every head and feed-forward width is padded to a multiple of eight with zero weights, which changes nothing and keeps
all operands 16-byte aligned.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..models.potodra import AttentionConfig, DenseConfig, MlstmConfig, ParallelConfig, PotodraConfig
from ..ops import moe, native, recurrent, stream, window
from ..ops.latent import prefill_items
from ..ops.stream import pad8, pad_heads, pad_to
from .batch import StepBatch
from .cache import HybridCache

SHORT_PORTION = 8
UNIT_SLOPE, UNIT_SHIFT = 1.702, 1.0      # gated units of experts: g sigmoid(1.702 g) (u + 1)


class _Weights:
    """Fields of one sub-layer, set by its loader."""


class _Step:
    """What one batch's sub-layers share."""

    def __init__(self, batch: StepBatch, cache: HybridCache, tabs, items):
        self.batch, self.cache, self.tabs, self.items = batch, cache, tabs, items
        self._chunks: dict = {}

    def chunks(self, size: int) -> recurrent.Chunks:
        """The batch's long portions in chunks of ``size`` tokens."""
        if size not in self._chunks:
            self._chunks[size] = recurrent.cut([(g.row0, g.n) for g in self.batch.segments], size, self.cache.state.device)
        return self._chunks[size]

    def portions(self, chunked: bool):
        """(portions that go token by token, portions that go in chunks or None)."""
        b = self.batch
        return (b.seqs[:b.n_short], b.seqs[b.n_short:]) if chunked and b.segments else (b.seqs, None)


class PotodraServing:
    tensor_parallel = False

    def __init__(self, cfg, device, rank: int = 0, world: int = 1, seed: int = 0,
                 weights: Optional[Dict[str, torch.Tensor]] = None):
        m: PotodraConfig = cfg.model
        self.cfg, self.model, self.device = cfg, m, torch.device(device)
        if self.device.type != "cuda":
            raise RuntimeError("Potodra is served by CUDA kernels; it has no CPU path")
        if cfg.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"Potodra is served in bfloat16 or float32, not {cfg.dtype}")
        self._check_sizes(m)
        self.vocab_local = m.vocab_size
        self.exact = cfg.dtype == torch.float32      # 32-bit everywhere: no tensor cores
        if weights is None:
            weights = m.random_weights(seed, device=self.device)
        m.check_weights(weights)
        self.weights = weights
        self.dp = pad8(m.d_model)
        self.side = torch.cuda.Stream(self.device)   # the experts of a small batch run beside the shared one
        self.rotations: list = []                    # distinct rotations: (spec, frequencies, factor)
        emb = self._get("embed")
        self.emb = emb.contiguous()
        self.head = pad_to(emb, m.vocab_size, self.dp).contiguous()
        self.subs: List[_Weights] = []
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
    def _check_sizes(m: PotodraConfig) -> None:
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
    def _get(self, name: str) -> torch.Tensor:
        return self.weights[name].to(device=self.device, dtype=self.cfg.dtype)

    def _f32(self, name: str) -> torch.Tensor:
        return self.weights[name].to(device=self.device, dtype=torch.float32).contiguous()

    def _add(self, layer: int, q: int, s: _Weights) -> None:
        p = f"l{layer}."
        s.layer, s.norm = layer, self._f32(f"{p}norm{q}")
        s.hc_in, s.hc_out, s.hc_mix = (self._f32(f"{p}hc{q}.{k}") for k in ("in", "out", "mix"))
        self.subs.append(s)

    def _heads(self, name: str, heads: int, size: int) -> torch.Tensor:
        """A projection's rows by head, padded."""
        return pad_heads(self._get(name), heads, (size,), self.dp)

    def _head_columns(self, name: str, heads: int, size: int) -> torch.Tensor:
        """An output projection's columns by head, padded."""
        return pad_heads(self._get(name).t(), heads, (size,), self.model.d_model).t()

    def _by_head(self, t: torch.Tensor, heads: int, size: int) -> torch.Tensor:
        return pad_heads(t.view(-1, 1), heads, (size,), 1).view(-1).contiguous()

    def _attention_rows(self, s: _Weights, p: str, a: AttentionConfig, out_scale: float):
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

    def _load_attention(self, p: str, a: AttentionConfig) -> _Weights:
        s = _Weights()
        s.run = self._attention
        rows, bias = self._attention_rows(s, p, a, 1.0)
        s.w_in, s.b_in = torch.cat(rows).contiguous(), torch.cat(bias).contiguous()
        s.w_out = self._head_columns(p + "o", a.heads, a.vdim).contiguous()
        return s

    def _load_mlstm(self, p: str, c: MlstmConfig) -> _Weights:
        s = _Weights()
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

    def _load_parallel(self, p: str, c: ParallelConfig) -> _Weights:
        s, r, left, right = _Weights(), c.right, p + "left.", p + "right."
        s.run, s.delta = self._parallel, r
        rows, bias = self._attention_rows(s, left, c.left, c.left_scale)
        H, G, d, e = r.heads, r.kv_heads, pad8(r.dim), pad8(r.vdim)
        parts = (("q", G, r.dim), ("k", G, r.dim), ("v", H, r.vdim))
        s.raw_col = sum(x.shape[0] for x in rows)
        rows += [self._heads(right + k, n, size) for k, n, size in parts]
        s.taps = torch.cat([pad_heads(self._f32(f"{right}{k}.conv"), n, (size,), r.conv) for k, n, size in parts]).t().contiguous()
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
        s.decay = torch.exp(self._f32(right + "A_log"))
        s.head_norm = pad_to(self._f32(right + "norm"), e) * c.right_scale
        s.w_out = torch.cat([self._head_columns(left + "o", c.left.heads, c.left.vdim), self._head_columns(right + "o", H, r.vdim)],
                            1).contiguous()
        s.chunked = recurrent.delta_chunks_covered(self.cfg.dtype, d, e)
        s.state = {"S": ((H, d, e), torch.float32), "conv": ((H, r.conv - 1, 2 * d + e), self.cfg.dtype)}
        return s

    def _load_dense(self, p: str, c: DenseConfig) -> _Weights:
        s, ff = _Weights(), pad8(c.ff)
        s.run = self._dense
        s.w_up = pad_to(self._get(p + "up"), ff, self.dp).contiguous()
        s.w_down = pad_to(self._get(p + "down"), self.model.d_model, ff).contiguous()
        return s

    def _load_mixture(self, p: str, c) -> _Weights:
        s, dp, D = _Weights(), self.dp, self.model.d_model
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

    def _rotation(self, spec) -> int:
        specs = [r[0] for r in self.rotations]
        if spec not in specs:
            freq, factor = spec.frequencies()
            self.rotations.append((spec, freq.to(self.device), factor))
            specs.append(spec)
        return specs.index(spec)

    # ------------------------------------------------------------------ what the engine calls
    @property
    def rows_per_portion(self) -> Optional[int]:
        """Portions up to this length run token by token through the row kernels, longer ones in tiles of queries.
        None: all of them by rows (32-bit, or sizes the prompt kernels do not cover)."""
        return SHORT_PORTION if self.tiled_prompts else None

    def max_positions(self) -> int:
        return self.cfg.num_blocks * self.cfg.block_size

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
        items = None
        if batch.segments:
            segs = [(s.row0, s.n, i, s.start) for i, s in enumerate(batch.segments)]
            items = torch.tensor(prefill_items(segs), dtype=torch.int32).to(self.device)
        st = _Step(batch, cache, [stream.rotary_table(batch.positions, f, s) for _, f, s in self.rotations], items)
        first = self.subs[0]
        h, x = stream.stream_mix_norm(x, first.hc_in, first.norm, eps, dt, self.dp)
        for i, s in enumerate(self.subs):
            y, rows = s.run(s, h, st)
            last = i + 1 == len(self.subs)
            w_in, norm = (self.sum, self.norm_f) if last else (self.subs[i + 1].hc_in, self.subs[i + 1].norm)
            h, x = stream.stream_mix_norm(x, w_in, norm, eps, dt, self.dp, y=y, mix=s.hc_mix, w_out=s.hc_out, add=rows, keep=not last)
        return h

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        """fp32 logits of normed rows."""
        return self._mm(hidden, self.head, out_dtype=torch.float32)

    # ------------------------------------------------------------------ sub-layers: input -> (fp32 result, rows to add to it)
    def _mm(self, a: torch.Tensor, w: torch.Tensor, **kw) -> torch.Tensor:
        """``a @ w.T`` for a weight stored ``[out, in]``."""
        return native.gemm(a, w.t(), path=2 if self.exact else 0, **kw)

    def _out(self, a: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        return self._mm(a, w, out_dtype=torch.float32)

    def _few(self, s: _Weights, h: torch.Tensor) -> torch.Tensor:
        """The numbers that drive a recurrence, in fp32."""
        if h.shape[0] <= recurrent.FEW_ROWS:
            return recurrent.few_outputs(h, s.w_few, s.b_few32)
        return self._mm(h, s.w_few, bias=s.b_few, out_dtype=torch.float32)

    def _heads_buffer(self, h: torch.Tensor, cols: int) -> torch.Tensor:
        return torch.empty((h.shape[0], cols), dtype=h.dtype, device=self.device)

    def _attend(self, s: _Weights, proj: torch.Tensor, out: torch.Tensor, st: _Step) -> None:
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

    def _attention(self, s: _Weights, h: torch.Tensor, st: _Step):
        proj = self._mm(h, s.w_in, bias=s.b_in)
        out = self._heads_buffer(h, s.o_cols)
        self._attend(s, proj, out, st)
        return self._out(out, s.w_out), None

    def _mlstm(self, s: _Weights, h: torch.Tensor, st: _Step):
        c = s.mlstm
        gates, proj = self._few(s, h), self._mm(h, s.w_in)
        out = self._heads_buffer(h, s.o_cols)
        rest = (st.cache.state[s.layer], proj[:, s.g_col:], s.head_norm, out, c.dim, c.vdim, c.gate_cap, self.model.norm_eps)
        short, long = st.portions(s.chunked)
        recurrent.mlstm_rows(proj, gates, short, *rest)
        if long is not None:
            recurrent.mlstm_chunks(proj, gates, st.chunks(recurrent.MLSTM_CHUNK), long, *rest)
        return self._out(out, s.w_out), None

    def _parallel(self, s: _Weights, h: torch.Tensor, st: _Step):
        r, state = s.delta, st.cache.state[s.layer]
        proj, few = self._mm(h, s.w_in, bias=s.b_in), self._few(s, h)
        out = self._heads_buffer(h, s.w_out.shape[1])
        self._attend(s, proj, out[:, :s.o_cols], st)
        (ac, an, a2), (gc, gn, g2) = s.low
        step, gate = self._out(proj[:, ac:ac + an], a2), self._mm(proj[:, gc:gc + gn], g2)
        raw = proj[:, s.raw_col:]
        inputs = (raw, s.taps, step, s.dt, s.decay, few)
        rest = (state, gate, s.head_norm, out[:, s.o_cols:], r.kv_heads, r.dim, r.vdim, self.model.norm_eps)
        short, long = st.portions(s.chunked)
        recurrent.delta_rows(*inputs, short, *rest)
        if long is not None:
            recurrent.delta_chunks(*inputs, st.chunks(recurrent.DELTA_CHUNK), long, *rest)
        return self._out(out, s.w_out), None

    def _dense(self, s: _Weights, h: torch.Tensor, st: _Step):
        return self._out(self._mm(h, s.w_up, act="relu2"), s.w_down), None

    def _mixture(self, s: _Weights, h: torch.Tensor, st: _Step):
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

    def _experts(self, s: _Weights, h: torch.Tensor):
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
