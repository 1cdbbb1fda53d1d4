"""Llama with INT4 (AWQ-layout) weights for the serving engine: weights, paged attention and the decoder stack.

Weights are INT4 group-128 with fp16 scales, sharded Megatron-style across the tensor-parallel group (qkv /
gate-up by output columns, out-proj / down by input rows on group boundaries); decode uses the streaming GEMV
or the fused W4A16 kernel, prefill the dequant + tcgen05 GEMM path.
"""
from __future__ import annotations

import math
from ctypes import c_float, c_int, c_void_p
from typing import List

import torch

from ..nn.quant import QuantizedTensor, qmatmul_int4
from ..ops import functional as F, native
from ..ops._lib import check, count_launch, ptr, stream_ptr
from .batch import StepBatch
from .cache import PagedKVCache

P, I, Fl = c_void_p, c_int, c_float
native.register_signature("rb_paged_decode_splits", [I])
native.register_signature("rb_paged_decode_attn", [I, P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, Fl, P])
native.register_signature("rb_paged_decode_attn_hm", [I, P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, Fl, P])


def paged_decode_attention(q, k_cache, v_cache, block_tables, ctx_lens, scale: float, max_ctx: int,
                           head_major: bool = False):
    """q [B, H, D]; returns [B, H, D].  ``head_major``: cache is [blocks, Hkv, block_size, D]."""
    B, H, D = q.shape
    Hkv = k_cache.shape[1] if head_major else k_cache.shape[2]
    bs = k_cache.shape[2] if head_major else k_cache.shape[1]
    if q.is_cuda:
        L = native.lib()
        splits = L.rb_paged_decode_splits(int(max_ctx))
        so = torch.empty((B, H, splits, D), dtype=torch.float32, device=q.device)
        sml = torch.empty((B, H, splits, 2), dtype=torch.float32, device=q.device)
        out = torch.empty_like(q)
        fn = L.rb_paged_decode_attn_hm if head_major else L.rb_paged_decode_attn
        check(fn(native.dtype_code(q.dtype), ptr(q), ptr(k_cache), ptr(v_cache),
                 ptr(block_tables), ptr(ctx_lens), ptr(out), ptr(so), ptr(sml), B, H,
                 Hkv, D, bs, block_tables.shape[1], splits,
                 float(scale), stream_ptr()), "rb_paged_decode_attn")
        count_launch(2)
        return out
    outs = []
    for b in range(B):
        n = int(ctx_lens[b])
        idx = torch.arange(n)
        blk = block_tables[b, idx // bs].long()
        if head_major:
            kk, vv = k_cache[blk, :, idx % bs].float(), v_cache[blk, :, idx % bs].float()
        else:
            kk, vv = k_cache[blk, idx % bs].float(), v_cache[blk, idx % bs].float()   # [n, Hkv, D]
        rep = H // Hkv
        kk, vv = kk.repeat_interleave(rep, 1), vv.repeat_interleave(rep, 1)
        s = torch.einsum("hd,nhd->hn", q[b].float(), kk) * scale
        outs.append(torch.einsum("hn,nhd->hd", torch.softmax(s, -1), vv).to(q.dtype))
    return torch.stack(outs)


def _rope(x, positions, heads, hd, theta):
    """x [T, heads*hd] rotated in place by absolute positions [T]."""
    T = x.shape[0]
    if x.is_cuda:
        native.rope_(x, T, 1, heads, hd, 0, theta, False, pos_ids=positions)
        return x
    xr = x.view(T, heads, hd).float()
    half = hd // 2
    inv = theta ** (-2.0 * torch.arange(half, dtype=torch.float32) / hd)
    ang = positions.float()[:, None] * inv[None]
    cs, sn = ang.cos()[:, None, :], ang.sin()[:, None, :]
    a, b = xr[..., :half], xr[..., half:]
    x.copy_(torch.cat([a * cs - b * sn, b * cs + a * sn], -1).reshape(T, heads * hd).to(x.dtype))
    return x


class _Layer:
    pass


class Int4LlamaShard:
    """This rank's shard of an INT4-quantised Llama: random-init weights generated per layer and
    quantised on the fly (``seed`` makes every rank draw the same full matrices before slicing)."""

    def __init__(self, cfg, device, rank: int = 0, world: int = 1, seed: int = 0, weights=None):
        if weights is not None:
            raise ValueError("the INT4 Llama is initialised at random; it reads no checkpoint")
        m = cfg.model
        self.cfg, self.device, self.rank, self.world = cfg, device, rank, world
        assert m.num_heads % world == 0 and m.num_kv_heads % world == 0
        hd = m.d_model // m.num_heads
        self.hd = hd
        self.h_local, self.hkv_local = m.num_heads // world, m.num_kv_heads // world
        # row-parallel K splits must fall on quantisation-group boundaries: the FFN width is padded with
        # zero columns (gate, up) / zero rows (down) to a multiple of world x group size, which leaves the
        # function unchanged (silu(0) * 0 = 0 meets zero rows).  Llama-7B: 11008 -> 11264 at 4 and 8 ranks.
        step = world * cfg.group_size
        ffn_pad = (m.ffn_dim + step - 1) // step * step if world > 1 else m.ffn_dim
        ffn_local = ffn_pad // world
        self.ffn_padded = ffn_pad
        assert (self.h_local * hd) % cfg.group_size == 0 or world == 1
        # full matrices are drawn (same seed on every rank, so the slices fit together) and
        # quantised on the device the shard lives on
        gdev = device if torch.device(device).type == "cuda" else "cpu"
        g = torch.Generator(device=gdev).manual_seed(seed)
        std = 0.02

        def rnd(*shape):
            return torch.randn(*shape, generator=g, device=gdev) * std

        def q(w):
            return QuantizedTensor.from_f32(w.contiguous(), cfg.group_size, cfg.scale_dtype).to(device)

        self.emb = rnd(m.vocab_size, m.d_model).to(cfg.dtype).to(device)
        self.layers: List[_Layer] = []
        r, W = rank, world
        for _ in range(m.num_layers):
            L = _Layer()
            wq, wk, wv = rnd(m.d_model, m.num_heads * hd), rnd(m.d_model, m.num_kv_heads * hd), \
                rnd(m.d_model, m.num_kv_heads * hd)
            ql, kl = self.h_local * hd, self.hkv_local * hd
            L.qkv = q(torch.cat([wq[:, r * ql:(r + 1) * ql], wk[:, r * kl:(r + 1) * kl],
                                 wv[:, r * kl:(r + 1) * kl]], dim=1))
            wo = rnd(m.num_heads * hd, m.d_model)
            L.out = q(wo[r * ql:(r + 1) * ql])
            wg, wu = rnd(m.d_model, m.ffn_dim), rnd(m.d_model, m.ffn_dim)
            if ffn_pad != m.ffn_dim:
                wg = torch.nn.functional.pad(wg, (0, ffn_pad - m.ffn_dim))
                wu = torch.nn.functional.pad(wu, (0, ffn_pad - m.ffn_dim))
            L.gate_up = q(torch.cat([wg[:, r * ffn_local:(r + 1) * ffn_local],
                                     wu[:, r * ffn_local:(r + 1) * ffn_local]], dim=1))
            wd = rnd(m.ffn_dim, m.d_model)
            if ffn_pad != m.ffn_dim:
                wd = torch.nn.functional.pad(wd, (0, 0, 0, ffn_pad - m.ffn_dim))
            L.down = q(wd[r * ffn_local:(r + 1) * ffn_local])
            L.ln1 = torch.ones(m.d_model, dtype=cfg.dtype, device=device)
            L.ln2 = torch.ones(m.d_model, dtype=cfg.dtype, device=device)
            self.layers.append(L)
        self.ln_f = torch.ones(m.d_model, dtype=cfg.dtype, device=device)
        vloc = m.vocab_size // world
        self.vocab_local = vloc
        self.head = rnd(m.d_model, m.vocab_size)[:, r * vloc:(r + 1) * vloc].contiguous().to(cfg.dtype).to(device)

    # ------------------------------------------------------------------ what the engine calls
    tensor_parallel = True
    rows_per_portion = 1      # portions of one token attend through the paged decode kernel

    def max_positions(self) -> int:
        return self.cfg.model.seq_len + 512

    def make_cache(self) -> PagedKVCache:
        return PagedKVCache(self.cfg, self.hkv_local, self.hd, self.device)

    def forward(self, batch: StepBatch, cache: PagedKVCache, row_parallel) -> torch.Tensor:
        """Hidden states ``[T, d]`` after the final norm.  ``row_parallel(h, weight, residual)`` is the engine's
        row-parallel product with the residual added."""
        m = self.cfg.model
        hd, H, Hkv, eps = self.hd, self.h_local, self.hkv_local, m.rms_eps
        scale = 1.0 / math.sqrt(hd)
        x = F.embedding(batch.tokens, self.emb)
        T = x.shape[0]
        for li, L in enumerate(self.layers):
            h = F.rms_norm(x, L.ln1, eps)
            qkv = qmatmul_int4(h, L.qkv)
            q = qkv[:, : H * hd]
            k = qkv[:, H * hd: (H + Hkv) * hd]
            v = qkv[:, (H + Hkv) * hd:]
            _rope(q, batch.positions, H, hd, m.rope_theta)
            _rope(k, batch.positions, Hkv, hd, m.rope_theta)
            cache.append(li, k, v, batch.slots)
            o = self._attend(li, q.reshape(T, H, hd), k.reshape(T, Hkv, hd), v.reshape(T, Hkv, hd), batch, cache, scale)
            x = row_parallel(o.reshape(T, H * hd).contiguous(), L.out, x)
            h2 = F.rms_norm(x, L.ln2, eps)
            gu = qmatmul_int4(h2, L.gate_up)
            x = row_parallel(F.swiglu(gu), L.down, x)
        return F.rms_norm(x, self.ln_f, eps)

    def _attend(self, li, q, k, v, batch: StepBatch, cache: PagedKVCache, scale: float):
        """Single tokens through the paged decode kernel; each prompt portion through FlashAttention, whole
        prompts on the keys just computed, continuations on the prefix gathered from the cache."""
        outs = []
        if batch.n_rows:
            outs.append(paged_decode_attention(q[:batch.n_rows].contiguous(), cache.k[li], cache.v[li], batch.tables,
                                               batch.ctx, scale, batch.max_ctx, head_major=cache.head_major))
        for i, s in enumerate(batch.segments):
            r = slice(s.row0, s.row0 + s.n)
            kk, vv = k[r], v[r]
            if s.start:
                kk, vv = cache.gather(li, batch.seg_tables[i].long(), torch.arange(s.start + s.n, device=q.device))
            outs.append(F.flash_attention(q[r][None], kk[None], vv[None], True, scale)[0])
        return outs[0] if len(outs) == 1 else torch.cat(outs)

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return native.gemm(hidden.contiguous(), self.head) if hidden.is_cuda else hidden @ self.head
