"""Recurrent mixers with a matrix state per head: typed wrappers of ``csrc/kernels/{recurrent,mlstm_chunk,delta_chunk}.cu``.

A batch's portions are rows of ``seqs`` (int32 ``[n, 4]`` on the device): first row, tokens, place of the sequence's
state, position of its first token.  State tensors have a leading dimension of places and stay fp32.  Sizes ending in
``_p`` are padded to multiples of eight with zeros.
"""
from __future__ import annotations

from ctypes import c_float, c_int, c_longlong, c_void_p
from dataclasses import dataclass
from typing import Optional

import torch

from . import native
from ._lib import check, count_launch, ptr, stream_ptr

P, LL, I, Fl = c_void_p, c_longlong, c_int, c_float
native.register_signature("rb_recurrent_blocks", [I, I])
native.register_signature("rb_mlstm_rows", [I, P, LL, P, LL, P, I, P, P, P, P, LL, P, P, LL, P, I, I, I, I, Fl, Fl, Fl, P])
native.register_signature("rb_delta_rows", [I, P, LL, P, P, P, LL, I, P, P, P, LL, P, I, P, P, LL, P, P, LL, P, I, I, I, I, I, I, Fl, Fl, I, P])
native.register_signature("rb_few_outputs", [I, P, LL, P, P, P, LL, I, I, P])

MAX_DIM = 512           # key size of a head
FEW_ROWS = 128          # up to this many tokens ``few_outputs`` beats a matrix product


def few_outputs(h: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """fp32 ``h @ w.T + bias`` for a weight with few rows (``bias`` fp32)."""
    T, N = h.shape[0], w.shape[0]
    out = torch.empty((T, N), dtype=torch.float32, device=h.device)
    check(native.lib().rb_few_outputs(native.dtype_code(h.dtype), ptr(h), h.stride(0), ptr(w), ptr(bias), ptr(out), T, w.shape[1], N,
                                      stream_ptr()), "rb_few_outputs")
    count_launch()
    return out


def _scratch(dim_p: int, vdim_p: int, like: torch.Tensor) -> Optional[torch.Tensor]:
    """Results before the output norm, when a head's columns do not fit one pass."""
    if native.lib().rb_recurrent_blocks(dim_p, vdim_p) == 1:
        return None
    return torch.empty(like.shape, dtype=torch.float32, device=like.device)


def mlstm_rows(proj: torch.Tensor, gates: torch.Tensor, seqs: torch.Tensor, state, gate: torch.Tensor, norm: torch.Tensor,
               out: torch.Tensor, dim: int, vdim: int, cap: float, eps: float) -> None:
    """Matrix memory with exponential gates, token by token.  ``proj`` rows start with queries, keys ``[heads, dim_p]``
    and values ``[heads, vdim_p]``; ``gates`` fp32 ``[T, 2 heads]``: input and forget gates before their cap; ``state``:
    tensors S ``[places, heads, dim_p, vdim_p]``, n, m.  Heads, divided by their root mean square, times ``norm`` and the
    sigmoid of ``gate`` (views ``[T, heads * vdim_p]``), go to ``out``."""
    S, n, m = state["S"], state["n"], state["m"]
    _, H, dim_p, vdim_p = S.shape
    if not seqs.shape[0]:
        return
    check(native.lib().rb_mlstm_rows(native.dtype_code(proj.dtype), ptr(proj), proj.stride(0), ptr(gates), gates.stride(0), ptr(seqs),
                                     seqs.shape[0], ptr(S), ptr(n), ptr(m), ptr(gate), gate.stride(0), ptr(norm), ptr(out), out.stride(0),
                                     ptr(_scratch(dim_p, vdim_p, out)), H, dim_p, vdim_p, vdim, dim ** -0.5, float(cap), float(eps),
                                     stream_ptr()), "rb_mlstm_rows")
    count_launch()


def delta_rows(raw: torch.Tensor, taps: torch.Tensor, a: torch.Tensor, dt: torch.Tensor, decay: torch.Tensor, b: torch.Tensor,
               seqs: torch.Tensor, state, gate: torch.Tensor, norm: torch.Tensor, out: torch.Tensor, kv_heads: int, dim: int, vdim: int,
               eps: float, per_head: bool = False, silu: bool = False) -> None:
    """Gated delta rule, token by token.  ``raw`` rows start with queries, keys ``[kv_heads, dim_p]`` and values ``[heads,
    vdim_p]``, the inputs of the convolutions with ``taps`` (fp32 ``[taps, channels]``, the last for the current token);
    ``a`` fp32 ``[T, heads * dim_p]`` and ``dt``: steps before their softplus; ``decay`` ``[heads]``: the factor on them;
    ``b`` fp32 ``[T, >= heads]``: write strengths before their sigmoid; ``state``: S ``[places, heads, dim_p, vdim_p]`` and
    conv ``[places, heads, taps - 1, 2 dim_p + vdim_p]``, the last inputs of a head's channels; ``norm`` ``[vdim_p]`` is
    shared by the heads; ``gate`` and ``out`` as in ``mlstm_rows``.  ``per_head``: a head's channels decay together, ``a``
    ``[T, >= heads]`` and ``dt`` ``[heads]``; ``silu``: the gate is silu(gate) instead of its sigmoid."""
    S = state["S"]
    _, H, dim_p, vdim_p = S.shape
    if not seqs.shape[0]:
        return
    check(native.lib().rb_delta_rows(native.dtype_code(raw.dtype), ptr(raw), raw.stride(0), ptr(taps), ptr(state["conv"]), ptr(a), a.stride(0),
                                     int(per_head), ptr(dt), ptr(decay), ptr(b), b.stride(0), ptr(seqs), seqs.shape[0], ptr(S), ptr(gate), gate.stride(0), ptr(norm),
                                     ptr(out), out.stride(0), ptr(_scratch(dim_p, vdim_p, out)), H, kv_heads, dim_p, vdim_p, vdim,
                                     taps.shape[0], dim ** -0.5, float(eps), int(silu), stream_ptr()), "rb_delta_rows")
    count_launch()


# ---------------------------------------------------------------- prompt portions in chunks
native.register_signature("rb_mlstm_chunk_ok", [I, I, I])
native.register_signature("rb_mlstm_chunk_scratch", [I, I])
native.register_signature("rb_mlstm_chunk", [I, P, LL, I, P, LL, P, I, P, P, I, P, P, P, P, LL, P, P, LL, P, I, I, I, I, Fl, Fl, Fl, P])

MLSTM_CHUNK = 128


@dataclass
class Chunks:
    """Portions cut into chunks of up to ``size`` tokens: ``items`` int32 ``[n, 4]`` (first row, tokens, portion), a
    portion's chunks neighbours; ``first`` int32 ``[portions + 1]``: the first chunk of every portion."""
    size: int
    items: torch.Tensor
    first: torch.Tensor


def cut(portions, size: int, device) -> Chunks:
    """``portions``: (first row, tokens) each."""
    items, first = [], [0]
    for i, (row0, n) in enumerate(portions):
        items += [(row0 + at, min(size, n - at), i, 0) for at in range(0, n, size)]
        first.append(len(items))
    both = torch.tensor([x for it in items for x in it] + first, dtype=torch.int32).to(device)
    return Chunks(size, both[:4 * len(items)].view(-1, 4), both[4 * len(items):])


def mlstm_chunks_covered(dtype: torch.dtype, dim_p: int, vdim_p: int) -> bool:
    return dtype == torch.bfloat16 and bool(native.lib().rb_mlstm_chunk_ok(native.DT_BF16, dim_p, vdim_p))


def mlstm_chunks(proj: torch.Tensor, gates: torch.Tensor, chunks: Chunks, seqs: torch.Tensor, state, gate: torch.Tensor,
                 norm: torch.Tensor, out: torch.Tensor, dim: int, vdim: int, cap: float, eps: float) -> None:
    """As ``mlstm_rows``, for portions ``seqs`` cut into ``chunks`` of ``MLSTM_CHUNK`` tokens."""
    S, n, m = state["S"], state["n"], state["m"]
    _, H, dim_p, vdim_p = S.shape
    N, L = chunks.items.shape[0], native.lib()
    L.rb_mlstm_chunk_scratch.restype = c_longlong
    assert chunks.size == MLSTM_CHUNK
    scratch = torch.empty(N * H * L.rb_mlstm_chunk_scratch(dim_p, vdim_p), dtype=torch.uint8, device=proj.device)
    check(L.rb_mlstm_chunk(native.dtype_code(proj.dtype), ptr(proj), proj.stride(0), proj.shape[0], ptr(gates), gates.stride(0),
                           ptr(chunks.items), N, ptr(seqs), ptr(chunks.first), seqs.shape[0], ptr(S), ptr(n), ptr(m), ptr(gate),
                           gate.stride(0), ptr(norm), ptr(out), out.stride(0), ptr(scratch), H, dim_p, vdim_p, vdim, dim ** -0.5,
                           float(cap), float(eps), stream_ptr()), "rb_mlstm_chunk")
    count_launch(3)


native.register_signature("rb_delta_chunk_ok", [I, I, I])
native.register_signature("rb_delta_chunk_scratch", [I, I])
native.register_signature("rb_delta_chunk", [I, P, LL, I, P, P, P, LL, I, P, P, P, LL, P, I, P, P, I, P, P, LL, P, P, LL, P, I, I, I, I, I, I, Fl, Fl, I, P])

DELTA_CHUNK = 64


def delta_chunks_covered(dtype: torch.dtype, dim_p: int, vdim_p: int) -> bool:
    return dtype == torch.bfloat16 and bool(native.lib().rb_delta_chunk_ok(native.DT_BF16, dim_p, vdim_p))


def delta_chunks(raw: torch.Tensor, taps: torch.Tensor, a: torch.Tensor, dt: torch.Tensor, decay: torch.Tensor, b: torch.Tensor,
                 chunks: Chunks, seqs: torch.Tensor, state, gate: torch.Tensor, norm: torch.Tensor, out: torch.Tensor, kv_heads: int, dim: int,
                 vdim: int, eps: float, per_head: bool = False, silu: bool = False) -> None:
    """As ``delta_rows``, for portions ``seqs`` cut into ``chunks`` of ``DELTA_CHUNK`` tokens."""
    S, L = state["S"], native.lib()
    _, H, dim_p, vdim_p = S.shape
    L.rb_delta_chunk_scratch.restype = c_longlong
    n = chunks.items.shape[0]
    assert chunks.size == DELTA_CHUNK
    scratch = torch.empty(n * H * L.rb_delta_chunk_scratch(dim_p, vdim_p), dtype=torch.uint8, device=raw.device)
    check(L.rb_delta_chunk(native.dtype_code(raw.dtype), ptr(raw), raw.stride(0), raw.shape[0], ptr(taps), ptr(state["conv"]), ptr(a), a.stride(0),
                           int(per_head), ptr(dt), ptr(decay), ptr(b), b.stride(0), ptr(chunks.items), n, ptr(seqs), ptr(chunks.first), seqs.shape[0], ptr(S), ptr(gate),
                           gate.stride(0), ptr(norm), ptr(out), out.stride(0), ptr(scratch), H, kv_heads, dim_p, vdim_p, vdim, taps.shape[0],
                           dim ** -0.5, float(eps), int(silu), stream_ptr()), "rb_delta_chunk")
    count_launch(3)
