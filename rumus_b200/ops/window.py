"""Sliding-window attention with grouped key/value heads over a paged cache: typed wrappers of
``csrc/kernels/{window_attention,window_decode,window_prefill}.cu``.

Head sizes ending in ``_p`` are padded to multiples of eight.  Pools are ``[blocks, kv_heads, block_size, size]``.
"""
from __future__ import annotations

from ctypes import c_float, c_int, c_longlong, c_void_p
from typing import Optional, Tuple

import torch

from . import native
from ._lib import check, count_launch, ptr, stream_ptr

P, LL, I, Fl = c_void_p, c_longlong, c_int, c_float
native.register_signature("rb_window_post", [I, P, LL, P, P, P, P, P, P, LL, I, I, I, I, I, I, I, I, Fl, P])
native.register_signature("rb_window_rows_splits", [I, I, I, I, I, I])
native.register_signature("rb_window_rows", [I, P, LL, P, P, P, P, P, P, LL, I, P, LL, P, P] + [I] * 10 + [Fl, Fl, Fl, P])
native.register_signature("rb_window_decode_ok", [I, I, I, I])
native.register_signature("rb_window_decode_splits", [I, I, I, I])
native.register_signature("rb_window_decode", [I, P, LL, P, P, I, P, P, P, P, LL, I, P, LL, P, P] + [I] * 10 + [Fl, Fl, Fl, P])
native.register_signature("rb_window_prefill_ok", [I, I, I, I])
native.register_signature("rb_window_prefill", [I, P, LL, P, P, I, P, P, I, P, P, LL, I, P, LL] + [I] * 9 + [Fl, Fl, Fl, P])

GATE_NONE, GATE_ELEMENT, GATE_HEAD = 0, 1, 2
MAX_HEAD = 512
UNBOUNDED = 1 << 30     # a window that never ends


def window_post(proj: torch.Tensor, slots: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor, heads: int, dim: int, *,
                tab: Optional[torch.Tensor] = None, rot: int = 0, norms: Optional[Tuple[torch.Tensor, torch.Tensor]] = None,
                eps: float = 0.0, neighbours: bool = False) -> None:
    """``proj`` rows start with queries ``[heads, dim_p]``, keys and values; keys and values go to the cache rows
    ``slots`` (-1: nowhere).  ``norms``: RMS norm of every query and key head over its ``dim`` numbers with these
    weights; ``tab``: then a rotation of its first ``rot`` numbers, element i with element i + rot / 2
    (``neighbours``: element 2i with 2i + 1).  Queries change in place."""
    _, G, bs, dim_p = k_pool.shape
    qn, kn = norms if norms is not None else (None, None)
    check(native.lib().rb_window_post(native.dtype_code(proj.dtype), ptr(proj), proj.stride(0), ptr(tab), ptr(qn), ptr(kn),
                                      ptr(slots), ptr(k_pool), ptr(v_pool), proj.shape[0], heads, G, dim, dim_p,
                                      v_pool.shape[3], rot if tab is not None else 0, int(neighbours), bs, float(eps), stream_ptr()),
          "rb_window_post")
    count_launch()


def _gate(gate: Optional[torch.Tensor], kind: int):
    return (None, 0, GATE_NONE) if gate is None else (ptr(gate), gate.stride(0), kind)


def decode_covered(dtype: torch.dtype, dim_p: int, vdim_p: int, block_size: int, scale: float) -> bool:
    """Whether the tensor-core row kernel takes these sizes (others run on the plain one)."""
    return dtype == torch.bfloat16 and scale > 0 and bool(
        native.lib().rb_window_decode_ok(native.DT_BF16, dim_p, vdim_p, block_size))


def window_rows_attention(q: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor, tables: torch.Tensor, ctx: torch.Tensor,
                          sink: Optional[torch.Tensor], gate: Optional[torch.Tensor], gate_kind: int, out: torch.Tensor,
                          window: int, scale: float, max_ctx: int, splits: int = 0, plain: bool = False, keep: int = 0,
                          cap: Optional[float] = None, out_scale: float = 1.0) -> None:
    """Every row attends through its own block table to the last ``window`` of its ``ctx`` keys: ``q [rows, H,
    dim_p]`` (view, heads side by side), ``out [rows, H * vdim_p]`` (view).  ``sink`` (fp32 ``[H]``) joins the
    denominators; the result is multiplied by the sigmoid of ``gate`` (per number or per head).  The sequence's first
    ``keep`` keys stay visible outside the window; ``cap``: scores s become cap tanh(s / cap); ``out_scale``: factor on
    the result."""
    rows, H, dim_p = q.shape
    nb, G, bs, vdim_p = v_pool.shape
    L, dt, keys = native.lib(), native.dtype_code(q.dtype), min(window + keep, max_ctx)
    plain = plain or not decode_covered(q.dtype, dim_p, vdim_p, bs, scale)
    if not splits:
        splits = L.rb_window_rows_splits(H, G, dim_p, vdim_p, rows, keys) if plain else L.rb_window_decode_splits(H, G, rows, keys)
    po = ml = None
    if splits > 1:
        po = torch.empty((rows, H, splits, vdim_p), dtype=torch.float32, device=q.device)
        ml = torch.empty((rows, H, splits, 2), dtype=torch.float32, device=q.device)
    pools = (ptr(k_pool), ptr(v_pool)) if plain else (ptr(k_pool), ptr(v_pool), nb)
    check((L.rb_window_rows if plain else L.rb_window_decode)(
        dt, ptr(q), q.stride(0), *pools, ptr(tables), ptr(ctx), ptr(sink), *_gate(gate, gate_kind), ptr(out), out.stride(0), ptr(po),
        ptr(ml), rows, H, G, dim_p, vdim_p, min(window, UNBOUNDED), keep, bs, tables.shape[1], splits, float(scale), float(cap or 0.0),
        float(out_scale), stream_ptr()), "rb_window_rows")
    count_launch(2 if splits > 1 else 1)


def prefill_covered(dtype: torch.dtype, dim_p: int, vdim_p: int, block_size: int, scale: float) -> bool:
    """Whether the tensor-core prompt kernel takes these sizes."""
    return dtype == torch.bfloat16 and scale > 0 and bool(
        native.lib().rb_window_prefill_ok(native.DT_BF16, dim_p, vdim_p, block_size))


def window_prefill(q: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor, tables: torch.Tensor, items: torch.Tensor,
                   sink: Optional[torch.Tensor], gate: Optional[torch.Tensor], gate_kind: int, out: torch.Tensor, window: int,
                   scale: float, keep: int = 0, cap: Optional[float] = None, out_scale: float = 1.0) -> None:
    """Attention of prompt portions whose keys and values are in the cache: ``q [T, H, dim_p]`` and ``out [T, H *
    vdim_p]`` (views), ``items`` int32 ``[n, 4]`` on the device: (first query row, rows <= 128, row of ``tables``,
    position of the first query).  ``keep``, ``cap`` and ``out_scale`` as for rows."""
    T, H, dim_p = q.shape
    nb, G, bs, vdim_p = v_pool.shape
    check(native.lib().rb_window_prefill(native.dtype_code(q.dtype), ptr(q), q.stride(0), ptr(k_pool), ptr(v_pool), nb,
                                         ptr(tables), ptr(items), items.shape[0], ptr(sink), *_gate(gate, gate_kind), ptr(out),
                                         out.stride(0), T, H, G, dim_p, vdim_p, min(window, UNBOUNDED), keep, bs, tables.shape[1],
                                         float(scale), float(cap or 0.0), float(out_scale), stream_ptr()), "rb_window_prefill")
    count_launch()
