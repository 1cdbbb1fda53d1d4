"""Nufupel for the serving engine: weights in the layout the kernels take, and the decoder stack.

A layer is x <- x + (attention(h) + ff(h)) with h = norm1 x; what follows from that here:

* queries, keys, values, output gate and the gate | up of the dense (or shared) feed-forward come out of one matrix
  product;
* attention heads and feed-forward activations land side by side in one buffer, so that one product with
  [W_o | W_down] adds both to the fp32 residual in its epilogue;
* the experts of a mixture work from the same h; what they leave for a token is added to the residual by the kernel
  that computes the next norm.

Every head and feed-forward width is padded to a multiple of eight with zero weights, which changes nothing and keeps
all operands 16-byte aligned.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..models.nufupel import MixtureConfig, NufupelConfig
from ..ops import moe, native, stream, window
from ..ops.latent import prefill_items
from ..ops.stream import pad8, pad_heads, pad_to
from .batch import StepBatch
from .cache import PagedWindowCache

SHORT_PORTION = 8


class _Layer:
    pass


class NufupelServing:
    tensor_parallel = False

    def __init__(self, cfg, device, rank: int = 0, world: int = 1, seed: int = 0,
                 weights: Optional[Dict[str, torch.Tensor]] = None):
        m: NufupelConfig = cfg.model
        self.cfg, self.model, self.device = cfg, m, torch.device(device)
        if self.device.type != "cuda":
            raise RuntimeError("Nufupel is served by CUDA kernels; it has no CPU path")
        if cfg.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"Nufupel is served in bfloat16 or float32, not {cfg.dtype}")
        for i, c in enumerate(m.layers):
            if max(c.mixer.dim, c.mixer.vdim) > window.MAX_HEAD:
                raise ValueError(f"layer {i}: heads of more than {window.MAX_HEAD} numbers")
        self.vocab_local = m.vocab_size
        self.exact = cfg.dtype == torch.float32      # 32-bit everywhere: no tensor cores
        if weights is None:
            weights = m.random_weights(seed, device=self.device)
        m.check_weights(weights)
        self.dp = pad8(m.d_model)
        self.side = torch.cuda.Stream(self.device)   # the experts of a small batch run beside its attention
        self.rotations: list = []                    # distinct rotations: (spec, frequencies, factor)
        self.emb = self._get(weights, "embed").contiguous()
        own = {i: self._load_layer(weights, i) for i, c in enumerate(m.layers) if c.owner == i}
        self.layers: List[_Layer] = [own[c.owner] for c in m.layers]
        self.tiled_prompts = all(window.prefill_covered(cfg.dtype, L.dim_p, L.vdim_p, cfg.block_size, L.cfg.scale)
                                 for L in self.layers)
        self.norm_f = 1.0 + self._f32(weights, "final.norm")      # norm weights are stored around zero
        self.head = pad_to(self._get(weights, "head"), m.vocab_size, self.dp).contiguous()

    # ------------------------------------------------------------------ weights
    def _get(self, weights, name: str) -> torch.Tensor:
        return weights[name].to(device=self.device, dtype=self.cfg.dtype)

    def _f32(self, weights, name: str) -> torch.Tensor:
        return weights[name].to(device=self.device, dtype=torch.float32).contiguous()

    def _load_layer(self, weights, i: int) -> _Layer:
        c, dp, D, p = self.model.layers[i], self.dp, self.model.d_model, f"l{i}."
        L, a = _Layer(), c.mixer
        L.cfg, L.index = a, i
        H, G = a.heads, a.kv_heads
        L.dim_p, L.vdim_p = pad8(a.dim), pad8(a.vdim)
        L.q_cols, L.o_cols = H * L.dim_p, H * L.vdim_p
        L.norm1 = 1.0 + self._f32(weights, p + "norm1")
        L.sink = self._f32(weights, p + "mix.sink")
        L.qk_norms = (self._f32(weights, p + "mix.q.norm"), self._f32(weights, p + "mix.k.norm")) if a.qk_norm else None
        L.rot_id = -1 if a.rot is None else self._rotation(a.rot)
        rows = [pad_heads(self._get(weights, p + "mix.q"), H, (a.dim,), dp),
                pad_heads(self._get(weights, p + "mix.k"), G, (a.dim,), dp),
                pad_heads(self._get(weights, p + "mix.v"), G, (a.vdim,), dp)]
        L.g_col = sum(r.shape[0] for r in rows)
        g = self._get(weights, p + "mix.g")
        L.g_kind = window.GATE_HEAD if a.gate_per_head else window.GATE_ELEMENT
        rows.append(pad_to(g, pad8(H), dp) if a.gate_per_head else pad_heads(g, H, (a.vdim,), dp))
        out = [pad_heads(self._get(weights, p + "mix.o").t(), H, (a.vdim,), D).t()]
        L.mixture = c.mlp if isinstance(c.mlp, MixtureConfig) else None
        L.ff_col, L.ff_p, L.act = sum(r.shape[0] for r in rows), 0, stream.GLU_GELU
        if c.mlp is not None:
            u, ff = (p + "mlp.shared.", c.mlp.shared_ff) if L.mixture else (p + "mlp.", c.mlp.ff)
            L.ff_p = pad8(ff)
            L.act = stream.GLU_SILU if L.mixture else stream.GLU_GELU
            rows += [pad_to(self._get(weights, u + k), L.ff_p, dp) for k in ("gate", "up")]
            out.append(pad_to(self._get(weights, u + "down"), D, L.ff_p))
        L.w_in = torch.cat(rows).contiguous()
        L.w_out = torch.cat(out, 1).contiguous()
        if L.mixture:
            E = L.mixture.experts
            L.router = pad_to(self._get(weights, p + "mlp.router"), E, dp).contiguous()
            L.router_b = self._f32(weights, p + "mlp.router.b")

            def experts(name, *shape):
                return torch.stack([pad_to(self._get(weights, f"{p}mlp.e{e}.{name}"), *shape) for e in range(E)])

            L.w_gu = moe.interleave(experts("gate", L.mixture.ff, dp), experts("up", L.mixture.ff, dp))
            L.eff_p = L.w_gu.shape[1] // 2
            L.w_dn = experts("down", D, L.eff_p)
            L.counts = torch.zeros(E + 1, dtype=torch.int32, device=self.device)
        return L

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
        """Portions up to this length run token by token through the row kernel, longer ones in tiles of queries.
        None: all of them by rows (32-bit, or sizes the prompt kernel does not cover)."""
        return SHORT_PORTION if self.tiled_prompts else None

    def max_positions(self) -> int:
        return self.cfg.num_blocks * self.cfg.block_size

    def make_cache(self) -> PagedWindowCache:
        return PagedWindowCache(self.cfg.num_blocks, self.cfg.block_size,
                                [(L.cfg.kv_heads, L.dim_p, L.vdim_p) for L in self.layers], self.cfg.dtype, self.device)

    def _mm(self, a: torch.Tensor, w: torch.Tensor, **kw) -> torch.Tensor:
        """``a @ w.T`` for a weight stored ``[out, in]``."""
        return native.gemm(a, w.t(), path=2 if self.exact else 0, **kw)

    def forward(self, batch: StepBatch, cache: PagedWindowCache, row_parallel=None) -> torch.Tensor:
        """Hidden states ``[T, d]`` after the last layer and the final norm (activation type)."""
        m, dt, eps = self.model, self.cfg.dtype, self.model.norm_eps
        T = batch.tokens.shape[0]
        x = stream.embed_scaled(batch.tokens, self.emb, m.embedding_scale)
        tabs = [stream.rotary_table(batch.positions, f, s) for _, f, s in self.rotations]
        items = None
        if batch.segments:
            segs = [(s.row0, s.n, i, s.start) for i, s in enumerate(batch.segments)]
            items = torch.tensor(prefill_items(segs), dtype=torch.int32).to(self.device)
        experts = None                   # what the previous layer's experts left, and which rows of it a token gains
        for li, L in enumerate(self.layers):
            a = L.cfg
            h = stream.rms_norm_stream(x, L.norm1, None, eps, dt, self.dp, add=experts)[0]
            beside = bool(L.mixture) and T <= moe.ROUTE_ROWS
            if beside:
                self.side.wait_stream(torch.cuda.current_stream(self.device))
                with torch.cuda.stream(self.side):
                    experts = self._experts(L, h)
            proj = self._mm(h, L.w_in)
            rot = dict(tab=tabs[L.rot_id], rot=a.rot.dims, norms=L.qk_norms, eps=eps) if a.rot is not None else {}
            window.window_post(proj, batch.slots, cache.k[li], cache.v[li], a.heads, a.dim, **rot)
            mix = torch.empty((T, L.o_cols + L.ff_p), dtype=dt, device=self.device)
            self._attend(L, proj, mix, batch, items, cache.k[li], cache.v[li])
            if L.ff_p:
                stream.glu(L.act, proj[:, L.ff_col:], mix[:, L.o_cols:])
            x = self._mm(mix, L.w_out, residual=x, out_dtype=torch.float32)
            if beside:
                # what either stream allocated is used by the other between a fork and the join that follows it
                torch.cuda.current_stream(self.device).wait_stream(self.side)
            else:
                experts = self._experts(L, h) if L.mixture else None
        return stream.rms_norm_stream(x, self.norm_f, None, eps, dt, self.dp, add=experts)[0]

    def _attend(self, L, proj, mix, batch: StepBatch, items, k_pool, v_pool) -> None:
        """Gated heads of every row into ``mix[:, :o_cols]``, from the cache that already holds this step's tokens."""
        a, T, n = L.cfg, proj.shape[0], batch.n_rows
        q = proj[:, :L.q_cols].unflatten(1, (a.heads, L.dim_p))
        gate, o = proj[:, L.g_col:], mix[:, :L.o_cols]
        if n:
            window.window_rows_attention(q[:n], k_pool, v_pool, batch.tables, batch.ctx, L.sink, gate, L.g_kind, o, a.window,
                                         a.scale, batch.max_ctx)
        if items is not None:
            window.window_prefill(q, k_pool, v_pool, batch.seg_tables, items, L.sink, gate, L.g_kind, o, a.window, a.scale)

    def _experts(self, L, h: torch.Tensor):
        """Weighted outputs of the chosen experts, one row per (token, choice), and the rows of every token."""
        E, top, T = L.mixture.experts, L.mixture.top, h.shape[0]
        logits = self._mm(h, L.router, out_dtype=torch.float32) if self.exact or T > moe.ROUTE_ROWS else None
        r = moe.route(h, L.router, L.router_b, L.counts, top, logits=logits, plain=self.exact)
        act = torch.empty((r.slots, L.eff_p), dtype=h.dtype, device=self.device)
        y = torch.empty((r.slots, self.dp), dtype=h.dtype, device=self.device)
        moe.grouped(h, L.w_gu, r, act, gated=True, plain=self.exact)
        moe.grouped(act, L.w_dn, r, y, gated=False, plain=self.exact)
        return y, r.slot_of

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        """fp32 logits of normed rows."""
        return stream.softcap_(self._mm(hidden, self.head, out_dtype=torch.float32), self.model.logit_softcap)
