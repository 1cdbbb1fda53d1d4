"""Around the mixers of decoders with an fp32 residual stream: scaled embedding, norms, gated units, rotation tables,
soft-capped logits.  Typed wrappers of ``csrc/kernels/residual_stream.cu`` and parts of ``elementwise.cu``.

Widths ending in ``_p`` are padded to multiples of eight (zeros), which keeps every row 16-byte aligned whatever the
model's sizes are.
"""
from __future__ import annotations

from ctypes import c_float, c_int, c_longlong, c_void_p
from typing import Optional, Tuple

import torch

from . import native
from ._lib import check, count_launch, ptr, stream_ptr

P, LL, I, Fl = c_void_p, c_longlong, c_int, c_float
native.register_signature("rb_embed_scaled", [I, P, P, P, LL, I, I, Fl, P])
native.register_signature("rb_rms_norm_stream", [I, P, P, P, P, P, LL, I, I, Fl, P, LL, P, I, P])
native.register_signature("rb_glu", [I, I, P, P, LL, I, LL, LL, Fl, Fl, Fl, P])
native.register_signature("rb_softcap", [P, LL, I, LL, Fl, P])
native.register_signature("rb_rotary_table", [P, P, P, LL, I, Fl, P])

GLU_CLAMPED, GLU_GELU, GLU_SILU = 0, 1, 2


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def pad_to(w: torch.Tensor, *shape: int) -> torch.Tensor:
    """``w`` in the corner of a zero tensor."""
    out = w.new_zeros(shape)
    out[tuple(slice(0, n) for n in w.shape)] = w
    return out


def pad_heads(w: torch.Tensor, heads: int, parts, cols: int) -> torch.Tensor:
    """``[heads * sum(parts), in]`` -> ``[heads * sum(pad8(parts)), cols]``."""
    w = w.view(heads, sum(parts), w.shape[1])
    pieces, at = [], 0
    for n in parts:
        pieces.append(pad_to(w[:, at:at + n], heads, pad8(n), cols))
        at += n
    return torch.cat(pieces, 1).flatten(0, 1)


def embed_scaled(ids: torch.Tensor, table: torch.Tensor, scale: float) -> torch.Tensor:
    """fp32 ``[T, D]`` rows ``table[ids] * scale``."""
    T, (V, D) = ids.shape[0], table.shape
    x = torch.empty((T, D), dtype=torch.float32, device=table.device)
    check(native.lib().rb_embed_scaled(native.dtype_code(table.dtype), ptr(ids), ptr(table), ptr(x), T, D, V, float(scale),
                                       stream_ptr()), "rb_embed_scaled")
    count_launch()
    return x


def rms_norm_stream(x: torch.Tensor, w1: torch.Tensor, w2: Optional[torch.Tensor], eps: float, dtype, ldy: int,
                    add: Optional[Tuple[torch.Tensor, torch.Tensor]] = None):
    """RMS norms of the fp32 rows of ``x`` with one or two weights, ``[T, ldy]`` each (zero beyond D).  ``add``:
    (rows, int32 ``[T, n]`` of row numbers) that ``x`` gains first, in place."""
    T, D = x.shape
    y1 = torch.empty((T, ldy), dtype=dtype, device=x.device)
    y2 = torch.empty((T, ldy), dtype=dtype, device=x.device) if w2 is not None else None
    rows, index = add if add is not None else (None, None)
    assert rows is None or (rows.dtype == dtype and index.dtype == torch.int32)
    check(native.lib().rb_rms_norm_stream(native.dtype_code(dtype), ptr(x), ptr(w1), ptr(w2), ptr(y1), ptr(y2), T, D, ldy,
                                          float(eps), ptr(rows), 0 if rows is None else rows.stride(0), ptr(index),
                                          0 if rows is None else index.shape[1], stream_ptr()), "rb_rms_norm_stream")
    count_launch()
    return y1, y2


def glu(kind: int, gu: torch.Tensor, out: torch.Tensor, limit: float = 0.0, slope: float = 0.0, shift: float = 0.0) -> None:
    """``gu``: ``[T, 2F]`` view laid out gate | up; ``out``: ``[T, F]`` view.  ``GLU_GELU``: gelu_tanh(gate) up;
    ``GLU_SILU``: silu(gate) up; ``GLU_CLAMPED``: see ``clamped_glu``."""
    T, F = out.shape
    check(native.lib().rb_glu(native.dtype_code(gu.dtype), kind, ptr(gu), ptr(out), T, F, gu.stride(0), out.stride(0),
                              float(limit), float(slope), float(shift), stream_ptr()), "rb_glu")
    count_launch()


def clamped_glu(gu: torch.Tensor, out: torch.Tensor, limit: float, slope: float, shift: float) -> None:
    """``out = g sigmoid(slope g) (u + shift)`` with ``g = min(gate, limit)``, ``u = clamp(up, -limit, limit)``."""
    glu(GLU_CLAMPED, gu, out, limit, slope, shift)


def softcap_(logits: torch.Tensor, cap: float) -> torch.Tensor:
    """fp32 ``[n, V]`` logits <- cap tanh(logits / cap)."""
    n, V = logits.shape
    check(native.lib().rb_softcap(ptr(logits), n, V, logits.stride(0), float(cap), stream_ptr()), "rb_softcap")
    count_launch()
    return logits


def rotary_table(positions: torch.Tensor, freq: torch.Tensor, mscale: float) -> torch.Tensor:
    """fp32 ``[T, pairs, 2]``: cos and sin of position x frequency, times ``mscale``."""
    T, n = positions.shape[0], freq.shape[0]
    tab = torch.empty((T, n, 2), dtype=torch.float32, device=positions.device)
    check(native.lib().rb_rotary_table(ptr(positions), ptr(freq), ptr(tab), T, n, float(mscale), stream_ptr()), "rb_rotary_table")
    count_launch()
    return tab
