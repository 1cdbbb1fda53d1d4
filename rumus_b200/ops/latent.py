"""Attention over key/value latents: typed wrappers of
``csrc/kernels/{latent_attention,latent_prefill,latent_decode}.cu``.

Widths ending in ``_p`` are padded to multiples of eight (zeros), which keeps every row 16-byte aligned
whatever the model's sizes are.
"""
from __future__ import annotations

from ctypes import c_float, c_int, c_longlong, c_void_p
from typing import List, Optional

import torch

from . import native
from ._lib import check, count_launch, ptr, stream_ptr
from .stream import clamped_glu, embed_scaled, pad8, rms_norm_stream, rotary_table  # noqa: F401

P, LL, I, Fl = c_void_p, c_longlong, c_int, c_float
native.register_signature("rb_latent_post", [I, P, LL, P, P, P, P, LL, I, I, I, I, I, I, I, Fl, P])
native.register_signature("rb_latent_gather", [P, P, P, P, I, I, I, I, LL, P])
native.register_signature("rb_latent_rows_attn", [I, P, P, LL, I, P, P, P, P, P, P, P, I, I, I, I, I, I, I, Fl, P])
native.register_signature("rb_sigmoid_gate", [I, P, LL, P, LL, LL, I, P])
native.register_signature("rb_latent_merge", [I, P, P, P, P, I, I, I, I, P])
native.register_signature("rb_latent_decode_ok", [I, I, I, I, I])
native.register_signature("rb_latent_decode_splits", [I, I, I, I, I])
native.register_signature("rb_latent_decode", [I, P, P, LL, I, P, I, P, P, P, P, I, I, I, I, I, I, I, Fl, P])
native.register_signature("rb_head_gemm", [I, P, LL, LL, P, I, P, LL, LL, P, LL, LL, I, I, I, I, P])
native.register_signature("rb_latent_prefill_ok", [I, I, I, I])
native.register_signature("rb_latent_prefill", [I, P, LL, P, LL, P, LL, P, I, P, P, LL, P, LL, I, I, I, I, I, I, I, Fl, P])


def latent_post(proj: torch.Tensor, tab: torch.Tensor, heads: int, dim_p: int, rot: int, *, kv_col: int = -1,
                norm_w: Optional[torch.Tensor] = None, slots: Optional[torch.Tensor] = None,
                pool: Optional[torch.Tensor] = None, rank: int = 0, eps: float = 0.0) -> None:
    """Rotates the queries' rotated parts of ``proj`` in place; with ``kv_col`` also norms the latent that starts
    at that column, rotates the shared key part behind it and writes both to the cache rows ``slots``."""
    check(native.lib().rb_latent_post(native.dtype_code(proj.dtype), ptr(proj), proj.stride(0), ptr(tab), ptr(norm_w),
                                      ptr(slots), ptr(pool), proj.shape[0], heads, dim_p, rot, pad8(rot), kv_col, rank,
                                      pad8(rank), float(eps), stream_ptr()), "rb_latent_post")
    count_launch()


def latent_gather(pool: torch.Tensor, tables: torch.Tensor, seg_off: torch.Tensor, total: int) -> torch.Tensor:
    """Cache rows of several prefixes one behind the other, ``[total, row]``."""
    out = torch.empty((total, pool.shape[2]), dtype=pool.dtype, device=pool.device)
    check(native.lib().rb_latent_gather(ptr(pool), ptr(tables), ptr(seg_off), ptr(out), tables.shape[0], tables.shape[1],
                                        pool.shape[1], pool.shape[2] * pool.element_size(), total, stream_ptr()),
          "rb_latent_gather")
    count_launch()
    return out


def head_matmul(a: torch.Tensor, w: torch.Tensor, out: torch.Tensor, transposed: bool,
                gate: Optional[torch.Tensor] = None, plain: bool = False) -> None:
    """One product per head: ``out[:, h] = a[:, h] @ (w[h].T if transposed else w[h])``, times ``sigmoid(gate[:, h])``;
    ``a``, ``out`` and ``gate`` are ``[T, H, *]`` views with contiguous last dimension.  16-bit operands run on the
    tensor cores unless ``plain``."""
    T, H, K = a.shape
    N = out.shape[2]
    if a.dtype == torch.bfloat16 and not plain:
        g = (ptr(gate), gate.stride(0), gate.stride(1)) if gate is not None else (None, 0, 0)
        check(native.lib().rb_head_gemm(native.dtype_code(a.dtype), ptr(a), a.stride(0), a.stride(1), ptr(w), 0 if transposed else 1,
                                        ptr(out), out.stride(0), out.stride(1), *g, T, H, K, N, stream_ptr()), "rb_head_gemm")
        count_launch()
        return
    check(native.lib().rb_bmm_simt(native.dtype_code(a.dtype), 0, 0 if transposed else 1, ptr(a), a.stride(0), a.stride(1),
                                   ptr(w), w.stride(1), w.stride(0), H, T, N, K, ptr(out), out.stride(0), out.stride(1), 0,
                                   1.0, stream_ptr()), "rb_bmm_simt")
    count_launch()
    if gate is not None:
        sigmoid_gate_(out, gate)


def decode_covered(dtype: torch.dtype, heads: int, rank_p: int, rot_p: int, block_size: int, scale: float) -> bool:
    """Whether the tensor-core decode kernel takes these sizes (others run on the plain kernel)."""
    return dtype == torch.bfloat16 and scale > 0 and bool(
        native.lib().rb_latent_decode_ok(native.DT_BF16, heads, rank_p, rot_p, block_size))


def prefill_covered(dtype: torch.dtype, dim_p: int, rot_p: int, vdim_p: int, scale: float) -> bool:
    """Whether the tensor-core prompt kernel takes these sizes."""
    return dtype == torch.bfloat16 and scale > 0 and bool(native.lib().rb_latent_prefill_ok(native.DT_BF16, dim_p, rot_p, vdim_p))


def latent_rows_attention(qa: torch.Tensor, qr: torch.Tensor, pool: torch.Tensor, tables: torch.Tensor, ctx: torch.Tensor,
                          sink: Optional[torch.Tensor], scale: float, max_ctx: int, plain: bool = False) -> torch.Tensor:
    """Each row attends through its own block table: ``qa [rows, H, rank_p]`` queries in latent space, ``qr
    [rows, H, rot_p]`` (a view) their rotated parts.  Returns the weighted sums of latents ``[rows, H, rank_p]``;
    ``sink`` (fp32 ``[H]``) joins the denominators."""
    rows, H, R = qa.shape
    rot_p, bs = qr.shape[2], pool.shape[1]
    L, dt = native.lib(), native.dtype_code(qa.dtype)
    plain = plain or not decode_covered(qa.dtype, H, R, rot_p, bs, scale)
    splits = max(1, min(16, (max_ctx + 511) // 512)) if plain else L.rb_latent_decode_splits(H, R, rot_p, rows, max_ctx)
    out = torch.empty_like(qa)
    po = torch.empty((rows, H, splits, R), dtype=torch.float32, device=qa.device)
    ml = torch.empty((rows, H, splits, 2), dtype=torch.float32, device=qa.device)
    if plain:
        check(L.rb_latent_rows_attn(dt, ptr(qa), ptr(qr), qr.stride(0), qr.stride(1), ptr(pool), ptr(tables), ptr(ctx), ptr(sink),
                                    ptr(out), ptr(po), ptr(ml), rows, H, R, rot_p, bs, tables.shape[1], splits, float(scale),
                                    stream_ptr()), "rb_latent_rows_attn")
    else:
        check(L.rb_latent_decode(dt, ptr(qa), ptr(qr), qr.stride(0), qr.stride(1), ptr(pool), pool.shape[0] * bs, ptr(tables),
                                 ptr(ctx), ptr(po), ptr(ml), rows, H, R, rot_p, bs, tables.shape[1], splits, float(scale),
                                 stream_ptr()), "rb_latent_decode")
        check(L.rb_latent_merge(dt, ptr(po), ptr(ml), ptr(sink), ptr(out), rows, H, R, splits, stream_ptr()), "rb_latent_merge")
    count_launch(2)
    return out


QUERY_TILE = 128


def prefill_items(segments) -> List[List[int]]:
    """Work items of ``latent_prefill``: tiles of up to 128 query rows of each portion, those with the most keys
    first.  ``segments``: (first row, rows, first key row, position of the first token)."""
    items = []
    for row0, n, key0, start in segments:
        for i in range(0, n, QUERY_TILE):
            items.append([row0 + i, min(QUERY_TILE, n - i), key0, start + i])
    return sorted(items, key=lambda it: -(it[3] + it[1]))


def latent_prefill(q: torch.Tensor, kv: torch.Tensor, rows: torch.Tensor, items: torch.Tensor, sink: Optional[torch.Tensor],
                   gate: Optional[torch.Tensor], out: torch.Tensor, dim_p: int, vdim_p: int, rank_p: int, scale: float) -> None:
    """Attention of prompt portions: ``q [T, H, dim_p + rot_p]`` (view), ``kv [keys, H dim_p + H vdim_p]`` expanded
    keys | values, ``rows [keys, rank_p + rot_p]`` the latent rows (the shared key part is read from them),
    ``items`` int32 ``[n, 4]`` on the device.  Gated heads go to ``out [T, >= H vdim_p]`` (view)."""
    T, H, dq = q.shape
    g = (ptr(gate), gate.stride(0)) if gate is not None else (None, 0)
    check(native.lib().rb_latent_prefill(native.dtype_code(q.dtype), ptr(q), q.stride(0), ptr(kv), kv.stride(0), ptr(rows),
                                         rows.stride(0), ptr(items), items.shape[0], ptr(sink), *g, ptr(out), out.stride(0), T,
                                         rows.shape[0], H, dim_p, dq - dim_p, vdim_p, rank_p, float(scale), stream_ptr()),
          "rb_latent_prefill")
    count_launch()


def sigmoid_gate_(x: torch.Tensor, g: torch.Tensor) -> None:
    """``x *= sigmoid(g)`` on ``[T, H, n]`` views whose heads lie side by side."""
    T, H, n = x.shape
    assert H == 1 or (x.stride(1) == n and g.stride(1) == n)
    check(native.lib().rb_sigmoid_gate(native.dtype_code(x.dtype), ptr(x), x.stride(0), ptr(g), g.stride(0), T, H * n,
                                       stream_ptr()), "rb_sigmoid_gate")
    count_launch()
