"""Mixture of experts: routing on the device and grouped products.  Typed wrappers of
``csrc/kernels/{moe,moe_gemm}.cu``."""
from __future__ import annotations

from ctypes import c_float, c_int, c_longlong, c_void_p
from dataclasses import dataclass
from typing import Optional

import torch

from . import native
from ._lib import check, count_launch, ptr, stream_ptr

P, LL, I, Fl = c_void_p, c_longlong, c_int, c_float
native.register_signature("rb_moe_route", [I, P, LL, P, I, P, LL] + [P] * 12 + [I] * 8 + [P])
native.register_signature("rb_moe_plain", [I, I, P, LL, P, P, LL, P, P, I, P, P, I, I, Fl, Fl, Fl, P])
native.register_signature("rb_moe_gemm", [I, I, P, LL, I, P, I, P, LL, P, P, I, I, P, P, I, I, Fl, Fl, Fl, P])
native.register_signature("rb_moe_pair", [I, I, P, LL, P, I, P, LL, P, P, I, P, I, I, Fl, Fl, Fl, P])

ROUTE_ROWS = 128        # up to this many tokens the routing kernel computes the logits itself


MAX_EXPERTS, MAX_GROUPS = 1024, 64
SOFTMAX, SIGMOID = 0, 1
SILU = (float("inf"), 1.0, 0.0)      # limit, slope, shift of a gated unit (see ``stream.clamped_glu``)

PAIR_TILE = 256         # rows of a work item of the CTA-pair product
PAIR_LOAD = 160         # tokens per expert from which it pays


@dataclass
class Routing:
    """Which expert's slot every (token, choice) got.  Slots of an expert are neighbours; a work item is up to
    ``tile`` of them."""
    tile: int
    max_items: int
    slots: int                   # rows of buffers by slot
    idx: torch.Tensor            # int32 [T, top]
    weight: torch.Tensor         # fp32 [T, top]
    slot_of: torch.Tensor        # int32 [T, top]
    slot_token: torch.Tensor     # int32 [slots]
    slot_weight: torch.Tensor    # fp32 [slots]
    items: torch.Tensor          # int32 [max_items, 4]: expert, first slot, slots
    n_items: torch.Tensor        # int32 [1]
    rows: Optional[torch.Tensor] = None     # [slots, dim] activations by slot (of large batches)


def interleave(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """``[E, F, dim]`` gates and ups -> ``[E, 2 F', dim]`` in the order the products take: 32 gates, 32 ups, ...;
    F' = F rounded up to 32 with zeros."""
    E, F, D = gate.shape
    out = gate.new_zeros((E, (F + 31) // 32, 2, 32, D))
    for i, w in enumerate((gate, up)):
        wide = gate.new_zeros((E, out.shape[1] * 32, D))
        wide[:, :F] = w
        out[:, :, i] = wide.view(E, -1, 32, D)
    return out.view(E, -1, D)


def slot_tile(pairs: int, experts: int, plain: bool) -> int:
    """Slots per work item: about what an expert gets when the load is even."""
    if plain:
        return 16
    if pairs >= PAIR_LOAD * experts:
        return PAIR_TILE
    tile = 16
    while tile < 128 and tile * experts < pairs:
        tile *= 2
    return tile


def route(h: torch.Tensor, router: torch.Tensor, bias: torch.Tensor, counts: torch.Tensor, top: int, *,
          logits: Optional[torch.Tensor] = None, plain: bool = False, tile: int = 0, score: int = SOFTMAX, groups: int = 1,
          keep: int = 1) -> Routing:
    """The ``top`` experts of every row of ``h [T, dim]`` by ``h @ router.T + bias`` (``logits``: the product
    without the bias, fp32 ``[T, >= E]``, if the caller has it) and the softmax over the chosen logits.
    ``score=SIGMOID``: the weights are the sigmoids of the logits without the bias, the choice goes by these plus the
    bias, among the ``keep`` best of ``groups`` groups of neighbours (by the sum of a group's two largest).
    ``counts``: int32 ``[E + 1]`` of zeros that the kernel leaves as zeros; ``plain``: the grouped products will be
    the plain ones."""
    T, E, dev = h.shape[0], bias.shape[0], h.device
    pairs = T * top
    tile = tile or slot_tile(pairs, E, plain)
    cap = min(E, pairs) + pairs // tile
    pair = tile == PAIR_TILE               # then item i is rows i * tile ... of buffers by slot
    slots = cap * tile if pair else pairs
    ints = torch.empty(3 * pairs + slots + E + 4 * cap + 4, dtype=torch.int32, device=dev)
    items, idx, rank, slot_of, slot_token, first, n_items = ints.split([4 * cap, pairs, pairs, pairs, slots, E, 4])
    fl = torch.empty(pairs + slots, dtype=torch.float32, device=dev)
    sort = pair or (T > ROUTE_ROWS and not plain)
    rows = torch.empty((slots, h.shape[1]), dtype=h.dtype, device=dev) if sort else None
    r = Routing(tile, cap, slots, idx.view(T, top), fl[:pairs].view(T, top), slot_of.view(T, top), slot_token, fl[pairs:],
                items.view(cap, 4), n_items[:1], rows)
    check(native.lib().rb_moe_route(native.dtype_code(h.dtype), ptr(h), h.stride(0), ptr(router), h.shape[1], ptr(logits),
                                    0 if logits is None else logits.stride(0), ptr(bias), ptr(counts), ptr(idx), ptr(fl), ptr(rank),
                                    ptr(first), ptr(items), ptr(r.n_items), ptr(slot_token), ptr(r.slot_weight), ptr(slot_of),
                                    ptr(rows), T, E, top, score, groups, keep, tile, tile if pair else 1, stream_ptr()), "rb_moe_route")
    count_launch(1 if pairs <= 4096 and not sort else 2)
    return r


def grouped(x: torch.Tensor, w: torch.Tensor, r: Routing, out: torch.Tensor, gated: bool, plain: bool = False, unit=SILU) -> torch.Tensor:
    """``gated``: ``out[slot] = weight unit(gate, up)`` of the slot's token, ``x [T, dim]``, ``w`` from ``interleave``;
    else ``out[slot] = w[e] x[slot]``, ``w [E, n, F]``, ``x [slots, F]``.  16-bit operands run on the tensor cores
    unless ``plain`` (which wants a routing made for it)."""
    E, n_out, n_in = w.shape
    n_out //= 2 if gated else 1
    L, dt = native.lib(), native.dtype_code(x.dtype)
    if plain:
        check(L.rb_moe_plain(dt, int(gated), ptr(x), x.stride(0), ptr(w), ptr(out), out.stride(0), ptr(r.items), ptr(r.n_items),
                             r.max_items, ptr(r.slot_token), ptr(r.slot_weight), n_in, n_out, *unit, stream_ptr()), "rb_moe_plain")
        count_launch()
        return out
    if gated and r.rows is not None:
        x = r.rows
    if r.tile == PAIR_TILE:
        check(L.rb_moe_pair(dt, int(gated), ptr(x), x.stride(0), ptr(w), E, ptr(out), out.stride(0), ptr(r.items), ptr(r.n_items),
                            r.max_items, ptr(r.slot_weight), n_in, n_out, *unit, stream_ptr()), "rb_moe_pair")
    else:
        check(L.rb_moe_gemm(dt, int(gated), ptr(x), x.stride(0), x.shape[0], ptr(w), E, ptr(out), out.stride(0), ptr(r.items),
                            ptr(r.n_items), r.max_items, r.tile, None if r.rows is not None else ptr(r.slot_token),
                            ptr(r.slot_weight), n_in, n_out, *unit, stream_ptr()), "rb_moe_gemm")
    count_launch()
    return out
