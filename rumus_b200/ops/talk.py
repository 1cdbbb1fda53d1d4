"""Attention whose heads mix their scores before the softmax (talking heads), over a paged cache of keys and of values:
typed wrappers of ``csrc/kernels/talk_*.cu``.

``mix`` is fp32 ``[H, H]``: head h's score is the sum over g of ``mix[h, g]`` times head g's.  Head sizes ending in ``_p``
are padded to multiples of eight.  Pools are ``[blocks, kv_heads, block_size, size]``.
"""
from __future__ import annotations

from ctypes import c_float, c_int, c_longlong, c_void_p
from typing import Optional

import torch

from . import native
from ._lib import check, count_launch, ptr, stream_ptr
from .window import UNBOUNDED, _gate

P, LL, I, Fl = c_void_p, c_longlong, c_int, c_float
native.register_signature("rb_talk_post", [I, P, LL, P, P, P, P, P, P, LL, I, I, I, I, I, I, P])
native.register_signature("rb_talk_rows_smem", [I, I, I])
native.register_signature("rb_talk_rows", [I, P, LL, P, P, P, P, P, P, P, LL, I, P, LL, P, P] + [I] * 9 + [Fl, P])
native.register_signature("rb_talk_decode_ok", [I] * 6)
native.register_signature("rb_talk_decode_splits", [I] * 5)
native.register_signature("rb_talk_decode", [I, P, LL, P, P, I, P, P, P, P, P, LL, I, P, LL, P, P] + [I] * 9 + [Fl, P])
native.register_signature("rb_talk_prefill_ok", [I] * 6)
native.register_signature("rb_talk_prefill", [I, P, I, I, P, P, I, P, P, I, P, P, LL, I, P, LL] + [I] * 7 + [Fl, P])

MAX_SMEM = 227 * 1024


def rows_covered(heads: int, dim_p: int, vdim_p: int) -> bool:
    """Whether any kernel takes all heads of a row at once."""
    return native.lib().rb_talk_rows_smem(heads, dim_p, vdim_p) <= MAX_SMEM


def talk_post(proj: torch.Tensor, slots: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor, mix: torch.Tensor, heads: int, rows: int, *,
              tab: Optional[torch.Tensor] = None, rot: int = 0) -> Optional[torch.Tensor]:
    """``proj`` rows start with queries ``[heads, dim_p]`` and keys; keys go to the cache rows ``slots`` (-1: nowhere),
    rotated (``tab``: the first ``rot`` numbers, element i with i + rot / 2), and unrotated as values.  The first ``rows``
    tokens' queries are rotated in place; the others' are rotated and mixed for ``talk_prefill``, ``[T - rows, heads, kv_heads,
    dim_p]`` (returned)."""
    T, (_, G, bs, dim_p) = proj.shape[0], k_pool.shape
    assert v_pool.shape == k_pool.shape
    qmix = torch.empty((T - rows, heads, G, dim_p), dtype=proj.dtype, device=proj.device) if rows < T else None
    check(native.lib().rb_talk_post(native.dtype_code(proj.dtype), ptr(proj), proj.stride(0), ptr(tab), ptr(slots), ptr(k_pool), ptr(v_pool),
                                    ptr(mix), ptr(qmix), T, rows, heads, G, dim_p, rot if tab is not None else 0, bs, stream_ptr()),
          "rb_talk_post")
    count_launch()
    return qmix


def talk_rows_attention(q: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor, tables: torch.Tensor, ctx: torch.Tensor, mix: torch.Tensor,
                        sink: Optional[torch.Tensor], gate: Optional[torch.Tensor], gate_kind: int, out: torch.Tensor, window: int, scale: float,
                        max_ctx: int, splits: int = 0, plain: bool = False) -> None:
    """Every row attends through its own block table to the last ``window`` of its ``ctx`` keys: ``q [rows, H, dim_p]``
    (view, heads side by side), ``out [rows, H * vdim_p]`` (view).  ``sink`` (fp32 ``[H]``) joins the denominators; the result
    is multiplied by the sigmoid of ``gate`` (per number or per head)."""
    rows, H, dim_p = q.shape
    nb, G, bs, vdim_p = v_pool.shape
    L, dt, keys = native.lib(), native.dtype_code(q.dtype), min(window, max_ctx)
    plain = plain or not L.rb_talk_decode_ok(dt, H, G, dim_p, vdim_p, bs)
    if not splits:
        splits = max(1, min(-(-keys // 64), 296 // rows)) if plain else L.rb_talk_decode_splits(H, G, dim_p, rows, keys)
    po = ml = None
    if splits > 1:
        po = torch.empty((rows, H, splits, vdim_p), dtype=torch.float32, device=q.device)
        ml = torch.empty((rows, H, splits, 2), dtype=torch.float32, device=q.device)
    pools = (ptr(k_pool), ptr(v_pool)) if plain else (ptr(k_pool), ptr(v_pool), nb)
    check((L.rb_talk_rows if plain else L.rb_talk_decode)(
        dt, ptr(q), q.stride(0), *pools, ptr(tables), ptr(ctx), ptr(mix), ptr(sink), *_gate(gate, gate_kind), ptr(out), out.stride(0), ptr(po),
        ptr(ml), rows, H, G, dim_p, vdim_p, min(window, UNBOUNDED), bs, tables.shape[1], splits, float(scale), stream_ptr()), "rb_talk_rows")
    count_launch(2 if splits > 1 else 1)


def prefill_covered(dtype: torch.dtype, heads: int, kv_heads: int, dim_p: int, vdim_p: int, block_size: int, scale: float) -> bool:
    """Whether the tensor-core prompt kernel takes these sizes."""
    return dtype == torch.bfloat16 and scale > 0 and bool(
        native.lib().rb_talk_prefill_ok(native.DT_BF16, heads, kv_heads, dim_p, vdim_p, block_size))


def talk_prefill(qmix: torch.Tensor, row0: int, k_pool: torch.Tensor, v_pool: torch.Tensor, tables: torch.Tensor, items: torch.Tensor,
                 sink: Optional[torch.Tensor], gate: Optional[torch.Tensor], gate_kind: int, out: torch.Tensor, window: int, scale: float) -> None:
    """Attention of prompt portions whose keys and values are in the cache: ``qmix`` from ``talk_post`` holds the queries of
    rows ``row0 ...`` of the batch, ``out [T, H * vdim_p]`` (view), ``items`` int32 ``[n, 4]`` on the device: (first query row,
    rows <= 128, row of ``tables``, position of the first query)."""
    n, H, G, dim_p = qmix.shape
    nb, _, bs, vdim_p = v_pool.shape
    check(native.lib().rb_talk_prefill(native.dtype_code(qmix.dtype), ptr(qmix), row0, n, ptr(k_pool), ptr(v_pool), nb, ptr(tables), ptr(items),
                                       items.shape[0], ptr(sink), *_gate(gate, gate_kind), ptr(out), out.stride(0), H, G, dim_p, vdim_p,
                                       min(window, UNBOUNDED), bs, tables.shape[1], float(scale), stream_ptr()), "rb_talk_prefill")
    count_launch()
