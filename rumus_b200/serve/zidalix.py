"""Zidalix for the serving engine: weights in the layout the kernels take, and the decoder stack.

A layer is x <- x + (attention(norm1 x) + ff(norm2 x)); what follows from that here:

* one kernel reads the fp32 residual and writes both normed copies;
* queries, latents and output gate come out of one matrix product, gate | up of the feed-forward out of another;
* attention heads and feed-forward activations land side by side in one buffer, so that one product with
  [W_o | W_down] finishes the layer and adds the residual in its epilogue.

Every head, latent and feed-forward width is padded to a multiple of eight with zero weights, which changes
nothing and keeps all operands 16-byte aligned.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..models.zidalix import ZidalixConfig
from ..ops import latent, native
from ..ops.stream import pad8, pad_heads, pad_to
from .batch import StepBatch
from .cache import PagedLatentCache

GLU_SLOPE, GLU_SHIFT = 1.702, 1.0
SHORT_PORTION = 8


class _Layer:
    pass


class ZidalixServing:
    tensor_parallel = False

    def __init__(self, cfg, device, rank: int = 0, world: int = 1, seed: int = 0,
                 weights: Optional[Dict[str, torch.Tensor]] = None):
        m: ZidalixConfig = cfg.model
        self.cfg, self.model, self.device = cfg, m, torch.device(device)
        if self.device.type != "cuda":
            raise RuntimeError("Zidalix is served by CUDA kernels; it has no CPU path")
        if cfg.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"Zidalix is served in bfloat16 or float32, not {cfg.dtype}")
        self.vocab_local = m.vocab_size
        self.exact = cfg.dtype == torch.float32      # 32-bit everywhere: no tensor cores
        if weights is None:
            weights = m.random_weights(seed, device=self.device)
        m.check_weights(weights)
        dt, D = cfg.dtype, m.d_model
        self.dp = dp = pad8(D)

        def get(name):
            return weights[name].to(device=self.device, dtype=dt)

        def f32(name):
            return weights[name].to(device=self.device, dtype=torch.float32).contiguous()

        self.emb = get("embed").contiguous()
        self.layers: List[_Layer] = []
        self.rotations: list = []                    # distinct rotations: (spec, frequencies, factor)
        for i, c in enumerate(m.layers):
            L, a, p = _Layer(), c.mixer, f"l{i}."
            L.cfg = a
            H = a.heads
            L.dim_p, L.rot_p, L.vdim_p, L.rank_p = pad8(a.dim), pad8(a.rot_dim), pad8(a.vdim), pad8(a.kv_rank)
            L.q_cols, L.o_cols = H * (L.dim_p + L.rot_p), H * L.vdim_p
            rows = [pad_heads(get(p + "mix.q"), H, (a.dim, a.rot_dim), dp)]
            L.kv_col, L.norm_kv = -1, None
            if a.kv_from is None:
                L.kv_col = L.q_cols
                rows.append(pad_heads(get(p + "mix.dkv"), 1, (a.kv_rank, a.rot_dim), dp))
                L.norm_kv = f32(p + "mix.dkv.norm")
            L.g_col = sum(r.shape[0] for r in rows)
            rows.append(pad_heads(get(p + "mix.g"), H, (a.vdim,), dp))
            L.w_in = torch.cat(rows).contiguous()
            # [H * dim_p + H * vdim_p, rank_p]: as a whole it writes keys and values out (prompts), by halves it
            # carries queries into latent space and weighted latents out of it (single tokens)
            L.ukv = torch.cat([pad_heads(get(p + "mix.uk"), H, (a.dim,), L.rank_p),
                               pad_heads(get(p + "mix.uv"), H, (a.vdim,), L.rank_p)]).contiguous()
            L.uk = L.ukv[:H * L.dim_p].view(H, L.dim_p, L.rank_p)
            L.uv = L.ukv[H * L.dim_p:].view(H, L.vdim_p, L.rank_p)
            L.sink = f32(p + "mix.sink")
            L.norm1, L.norm2 = f32(p + "norm1"), None
            out = [pad_heads(get(p + "mix.o").t(), H, (a.vdim,), D).t()]
            L.ff_p, L.limit = 0, 0.0
            if c.mlp is not None:
                L.norm2, L.ff_p, L.limit = f32(p + "norm2"), pad8(c.mlp.ff), c.mlp.limit
                L.w_gu = torch.cat([pad_to(get(p + "mlp.gate"), L.ff_p, dp), pad_to(get(p + "mlp.up"), L.ff_p, dp)]).contiguous()
                out.append(pad_to(get(p + "mlp.down"), D, L.ff_p))
            L.w_out = torch.cat(out, 1).contiguous()
            specs = [r[0] for r in self.rotations]
            if a.rot not in specs:
                freq, factor = a.rot.frequencies()
                self.rotations.append((a.rot, freq.to(self.device), factor))
                specs.append(a.rot)
            L.rot_id = specs.index(a.rot)
            self.layers.append(L)
        self.tiled_prompts = all(latent.prefill_covered(dt, L.dim_p, L.rot_p, L.vdim_p, L.cfg.scale) for L in self.layers)
        self.norm_f = f32("final.norm")
        self.head = pad_to(get("head"), m.vocab_size, dp).contiguous()

    # ------------------------------------------------------------------ what the engine calls
    @property
    def rows_per_portion(self) -> Optional[int]:
        """Portions up to this length run token by token through the decode kernels: for a few queries that costs
        less than writing every key and value of the prefix out.  None: all of them (32-bit, or sizes the prompt
        kernel does not cover)."""
        return SHORT_PORTION if self.tiled_prompts else None

    def max_positions(self) -> int:
        return self.cfg.num_blocks * self.cfg.block_size

    def make_cache(self) -> PagedLatentCache:
        rows = [L.rank_p + L.rot_p if L.kv_col >= 0 else 0 for L in self.layers]
        share = [i if L.cfg.kv_from is None else L.cfg.kv_from for i, L in enumerate(self.layers)]
        return PagedLatentCache(self.cfg.num_blocks, self.cfg.block_size, rows, share, self.cfg.dtype, self.device)

    def _mm(self, a: torch.Tensor, w: torch.Tensor, **kw) -> torch.Tensor:
        """``a @ w.T`` for a weight stored ``[out, in]``."""
        return native.gemm(a, w.t(), path=2 if self.exact else 0, **kw)

    def forward(self, batch: StepBatch, cache: PagedLatentCache, row_parallel=None) -> torch.Tensor:
        """fp32 residual stream ``[T, d]`` after the last layer, final norm applied (activation type)."""
        m, dt, eps = self.model, self.cfg.dtype, self.model.norm_eps
        T = batch.tokens.shape[0]
        x = latent.embed_scaled(batch.tokens, self.emb, m.embedding_scale)
        tabs = [latent.rotary_table(batch.positions, f, s) for _, f, s in self.rotations]
        plan = self._prompt_plan(batch)
        for li, L in enumerate(self.layers):
            a = L.cfg
            h1, h2 = latent.rms_norm_stream(x, L.norm1, L.norm2, eps, dt, self.dp)
            proj = self._mm(h1, L.w_in)
            own = dict(kv_col=L.kv_col, norm_w=L.norm_kv, slots=batch.slots, pool=cache.pool(li), rank=a.kv_rank, eps=eps) \
                if L.kv_col >= 0 else {}
            latent.latent_post(proj, tabs[L.rot_id], a.heads, L.dim_p, a.rot_dim, **own)
            mix = torch.empty((T, L.o_cols + L.ff_p), dtype=dt, device=self.device)
            self._attend(L, proj, mix, batch, plan, cache.pool(li))
            if L.ff_p:
                latent.clamped_glu(self._mm(h2, L.w_gu), mix[:, L.o_cols:], L.limit, GLU_SLOPE, GLU_SHIFT)
            x = self._mm(mix, L.w_out, residual=x, out_dtype=torch.float32)
        return latent.rms_norm_stream(x, self.norm_f, None, eps, dt, self.dp)[0]

    def _prompt_plan(self, batch: StepBatch):
        """(first key row of every portion's sequence in the gathered latents, their number, work items)."""
        if not batch.segments:
            return None
        off, segs = [0], []
        for s in batch.segments:
            segs.append((s.row0, s.n, off[-1], s.start))
            off.append(off[-1] + s.start + s.n)
        dev = self.device
        return (torch.tensor(off, dtype=torch.int32).to(dev), off[-1],
                torch.tensor(latent.prefill_items(segs), dtype=torch.int32).to(dev))

    def _attend(self, L, proj: torch.Tensor, mix: torch.Tensor, batch: StepBatch, plan, pool: torch.Tensor) -> None:
        """Gated heads of every row into ``mix[:, :o_cols]``.  Single tokens attend in latent space; for prompt
        portions the latents of their sequences are gathered and expanded to keys and values first."""
        a, T, n = L.cfg, proj.shape[0], batch.n_rows
        H = a.heads
        q = proj[:, :L.q_cols].view(T, H, L.dim_p + L.rot_p)
        gate = proj[:, L.g_col:].view(T, H, L.vdim_p)
        o = mix[:, :L.o_cols].unflatten(1, (H, L.vdim_p))
        if n:
            qa = torch.empty((n, H, L.rank_p), dtype=proj.dtype, device=proj.device)
            latent.head_matmul(q[:n, :, :L.dim_p], L.uk, qa, False)
            c = latent.latent_rows_attention(qa, q[:n, :, L.dim_p:], pool, batch.tables, batch.ctx, L.sink, a.scale, batch.max_ctx)
            latent.head_matmul(c, L.uv, o[:n], True, gate=gate[:n])
        if plan is not None:
            seg_off, keys, items = plan
            rows = latent.latent_gather(pool, batch.seg_tables, seg_off, keys)
            kv = self._mm(rows[:, :L.rank_p], L.ukv)
            latent.latent_prefill(q, kv, rows, items, L.sink, gate[:, 0], mix, L.dim_p, L.vdim_p, L.rank_p, a.scale)

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        """fp32 logits of normed rows."""
        return self._mm(hidden, self.head, alpha=self.model.logit_scale, out_dtype=torch.float32)
