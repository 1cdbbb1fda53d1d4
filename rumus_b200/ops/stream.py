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
native.register_signature("rb_glu", [I, I, P, P, LL, I, LL, LL, Fl, Fl, Fl, P, LL, P])
native.register_signature("rb_softcap", [P, LL, I, LL, Fl, P])
native.register_signature("rb_rotary_table", [P, P, P, LL, I, Fl, P])

native.register_signature("rb_stream_mix_norm", [I, P, LL, LL, P, P, P, P, P, P, P, LL, I, I, I, Fl, P, LL, P, I, P])
native.register_signature("rb_embed_norm", [I, P, P, P, P, I, P, P, LL, I, I, I, Fl, P])
native.register_signature("rb_scaled_add_norm", [I, P, P, P, P, I, P, LL, I, I, Fl, I, P])

MAX_STREAMS = 8
GLU_CLAMPED, GLU_GELU, GLU_SILU, GLU_RELU = 0, 1, 2, 3


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


def stream_mix_norm(x: torch.Tensor, w_in: torch.Tensor, w: torch.Tensor, eps: float, dtype, ldh: int, *,
                    y: Optional[torch.Tensor] = None, mix: Optional[torch.Tensor] = None, w_out: Optional[torch.Tensor] = None,
                    add: Optional[Tuple[torch.Tensor, torch.Tensor]] = None, keep: bool = True):
    """What lies between two sub-layers of a residual of parallel streams ``x`` (fp32 ``[T, streams, D]``; it may be a
    view whose streams are one): with the last sub-layer's result ``y`` (fp32 ``[T, D]``, plus the rows of ``add`` as in
    ``rms_norm_stream``) the streams become x_t = sum_s mix[s, t] x_s + w_out[t] y; the next one's input is the RMS norm
    with weight ``w`` of sum_s w_in[s] x_s, ``[T, ldh]`` of ``dtype``.  Returns (that, the new streams; None unless
    ``keep``).  ``x`` is overwritten when it can hold them."""
    T, S, D = x.shape
    h = torch.empty((T, ldh), dtype=dtype, device=x.device)
    xo = None
    if y is not None and keep:
        xo = x if x.is_contiguous() else torch.empty((T, S, D), dtype=torch.float32, device=x.device)
    rows, index = add if add is not None else (None, None)
    assert rows is None or (rows.dtype == dtype and index.dtype == torch.int32)
    assert y is None or (y.dtype == torch.float32 and y.is_contiguous())
    check(native.lib().rb_stream_mix_norm(native.dtype_code(dtype), ptr(x), x.stride(0), x.stride(1), ptr(xo), ptr(y), ptr(mix),
                                          ptr(w_out), ptr(w_in), ptr(w), ptr(h), T, S, D, ldh, float(eps), ptr(rows),
                                          0 if rows is None else rows.stride(0), ptr(index),
                                          0 if rows is None else index.shape[1], stream_ptr()), "rb_stream_mix_norm")
    count_launch()
    return h, (x if y is None and keep else xo)


def _step(w: torch.Tensor, D: int) -> int:
    """A norm's weight is a number per channel or one for all."""
    assert w.numel() in (1, D) and w.dtype == torch.float32
    return int(w.numel() > 1)


def embed_norm(ids: torch.Tensor, table: torch.Tensor, g: torch.Tensor, w: torch.Tensor, eps: float, ldh: int):
    """Embeddings that are normed: x = RMS norm of ``table[ids]`` times the number ``g`` (fp32 ``[T, D]``), and x's own RMS
    norm with weight ``w`` (``[D]`` or one number), ``[T, ldh]`` of the table's type (zero beyond D)."""
    T, (V, D) = ids.shape[0], table.shape
    x = torch.empty((T, D), dtype=torch.float32, device=table.device)
    h = torch.empty((T, ldh), dtype=table.dtype, device=table.device)
    check(native.lib().rb_embed_norm(native.dtype_code(table.dtype), ptr(ids), ptr(table), ptr(g), ptr(w), _step(w, D), ptr(x), ptr(h), T, D,
                                     ldh, V, float(eps), stream_ptr()), "rb_embed_norm")
    count_launch()
    return x, h


def scaled_add_norm(x: torch.Tensor, y: torch.Tensor, scale: torch.Tensor, w: torch.Tensor, eps: float, dtype, ldh: int,
                    keep: bool = True) -> torch.Tensor:
    """Between two sub-layers: ``x += scale * y`` (fp32 ``[T, D]``, ``scale`` per channel; in place if ``keep``, else only in
    what follows), and the RMS norm of the sum with weight ``w`` (``[D]`` or one number), ``[T, ldh]`` of ``dtype``."""
    T, D = x.shape
    h = torch.empty((T, ldh), dtype=dtype, device=x.device)
    assert x.is_contiguous() and y.is_contiguous() and y.dtype == torch.float32 and y.shape == x.shape and scale.numel() == D
    check(native.lib().rb_scaled_add_norm(native.dtype_code(dtype), ptr(x), ptr(y), ptr(scale), ptr(w), _step(w, D), ptr(h), T, D, ldh,
                                          float(eps), int(keep), stream_ptr()), "rb_scaled_add_norm")
    count_launch()
    return h


def glu(kind: int, gu: torch.Tensor, out: torch.Tensor, limit: float = 0.0, slope: float = 0.0, shift: float = 0.0,
        row_gate: Optional[torch.Tensor] = None) -> None:
    """``gu``: ``[T, 2F]`` view laid out gate | up; ``out``: ``[T, F]`` view.  ``GLU_GELU``: gelu_tanh(gate) up;
    ``GLU_SILU``: silu(gate) up; ``GLU_RELU``: max(gate, 0) up; ``GLU_CLAMPED``: see ``clamped_glu``.  ``row_gate`` (``[T, ...]`` view): rows are
    multiplied by the sigmoid of its first column."""
    T, F = out.shape
    check(native.lib().rb_glu(native.dtype_code(gu.dtype), kind, ptr(gu), ptr(out), T, F, gu.stride(0), out.stride(0),
                              float(limit), float(slope), float(shift), ptr(row_gate),
                              0 if row_gate is None else row_gate.stride(0), stream_ptr()), "rb_glu")
    count_launch()


def clamped_glu(gu: torch.Tensor, out: torch.Tensor, limit: float, slope: float, shift: float,
                row_gate: Optional[torch.Tensor] = None) -> None:
    """``out = g sigmoid(slope g) (u + shift)`` with ``g = min(gate, limit)``, ``u = clamp(up, -limit, limit)``."""
    glu(GLU_CLAMPED, gu, out, limit, slope, shift, row_gate)


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
