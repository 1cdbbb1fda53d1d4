"""Mixture of experts: routing on the device and grouped products.  Typed wrappers of
``csrc/kernels/{moe,moe_gemm}.cu``."""
from __future__ import annotations

from ctypes import c_int, c_longlong, c_void_p
from dataclasses import dataclass
from typing import Optional

import torch

from . import native
from ._lib import check, count_launch, ptr, stream_ptr

P, LL, I = c_void_p, c_longlong, c_int
native.register_signature("rb_moe_route", [I, P, LL, P, I, P, LL] + [P] * 11 + [I, I, I, I, P])
native.register_signature("rb_moe_plain", [I, I, P, LL, P, P, LL, P, P, I, P, P, I, I, P])
native.register_signature("rb_moe_gemm", [I, I, P, LL, I, P, I, P, LL, P, P, I, I, P, P, I, I, P])

ROUTE_ROWS = 128        # up to this many tokens the routing kernel computes the logits itself


@dataclass
class Routing:
    """Which expert's slot every (token, choice) got.  Slots of an expert are neighbours; a work item is up to
    ``tile`` of them."""
    tile: int
    max_items: int
    idx: torch.Tensor            # int32 [T, top]
    weight: torch.Tensor         # fp32 [T, top]
    slot_of: torch.Tensor        # int32 [T, top]
    slot_token: torch.Tensor     # int32 [T * top]
    slot_weight: torch.Tensor    # fp32 [T * top]
    items: torch.Tensor          # int32 [max_items, 4]: expert, first slot, slots
    n_items: torch.Tensor        # int32 [1]


def slot_tile(pairs: int, experts: int, plain: bool) -> int:
    """Slots per work item: about what an expert gets when the load is even."""
    if plain:
        return 16
    tile = 16
    while tile < 256 and tile * experts < pairs:
        tile *= 2
    return tile


def route(h: torch.Tensor, router: torch.Tensor, bias: torch.Tensor, counts: torch.Tensor, top: int, *,
          logits: Optional[torch.Tensor] = None, plain: bool = False) -> Routing:
    """The ``top`` experts of every row of ``h [T, dim]`` by ``h @ router.T + bias`` (``logits``: the product
    without the bias, fp32 ``[T, >= E]``, if the caller has it) and the softmax over the chosen logits.
    ``counts``: int32 ``[E + 1]`` of zeros that the kernel leaves as zeros; ``plain``: the grouped products will be
    the plain ones."""
    T, E, dev = h.shape[0], bias.shape[0], h.device
    pairs = T * top
    tile = slot_tile(pairs, E, plain)
    cap = min(E, pairs) + pairs // tile
    ints = torch.empty(4 * pairs + E + 4 * cap + 4, dtype=torch.int32, device=dev)
    items, idx, rank, slot_of, slot_token, first, n_items = ints.split([4 * cap, pairs, pairs, pairs, pairs, E, 4])
    fl = torch.empty(2 * pairs, dtype=torch.float32, device=dev)
    r = Routing(tile, cap, idx.view(T, top), fl[:pairs].view(T, top), slot_of.view(T, top), slot_token, fl[pairs:],
                items.view(cap, 4), n_items[:1])
    check(native.lib().rb_moe_route(native.dtype_code(h.dtype), ptr(h), h.stride(0), ptr(router), h.shape[1], ptr(logits),
                                    0 if logits is None else logits.stride(0), ptr(bias), ptr(counts), ptr(idx), ptr(fl), ptr(rank),
                                    ptr(first), ptr(items), ptr(r.n_items), ptr(slot_token), ptr(r.slot_weight), ptr(slot_of), T, E,
                                    top, tile, stream_ptr()), "rb_moe_route")
    count_launch(1 if pairs <= 4096 else 2)
    return r


def grouped(x: torch.Tensor, w: torch.Tensor, r: Routing, out: torch.Tensor, gated: bool, plain: bool = False) -> torch.Tensor:
    """``gated``: ``out[slot] = silu(gate) up`` of the slot's token, ``w [E, 2F, dim]`` gates then ups, ``x [T,
    dim]``; else ``out[slot] = weight (w[e] x[slot])``, ``w [E, n, F]``, ``x [slots, F]``.  16-bit operands run on
    the tensor cores unless ``plain`` (which wants a routing made for it)."""
    E, n_out, n_in = w.shape
    n_out //= 2 if gated else 1
    dt = native.dtype_code(x.dtype)
    if plain:
        check(native.lib().rb_moe_plain(dt, int(gated), ptr(x), x.stride(0), ptr(w), ptr(out), out.stride(0), ptr(r.items),
                                        ptr(r.n_items), r.max_items, ptr(r.slot_token), ptr(r.slot_weight), n_in, n_out,
                                        stream_ptr()), "rb_moe_plain")
    else:
        check(native.lib().rb_moe_gemm(dt, int(gated), ptr(x), x.stride(0), x.shape[0], ptr(w), E, ptr(out), out.stride(0),
                                       ptr(r.items), ptr(r.n_items), r.max_items, r.tile, ptr(r.slot_token), ptr(r.slot_weight),
                                       n_in, n_out, stream_ptr()), "rb_moe_gemm")
    count_launch()
    return out
