"""Block-paged caches.  All kinds share one block numbering (the scheduler's): token ``t`` of a sequence
lives at offset ``t % block_size`` of block ``table[t // block_size]`` in every layer's pool.  State of a fixed size per
sequence lives in slots beside them."""
from __future__ import annotations

from ctypes import c_int, c_longlong, c_void_p
from typing import Dict, List, Optional, Tuple

import torch

from ..ops import native
from ..ops._lib import check, count_launch, ptr, stream_ptr

P, LL, I = c_void_p, c_longlong, c_int
native.register_signature("rb_kv_append", [I, P, P, LL, P, P, P, I, I, P])
native.register_signature("rb_kv_append_hm", [I, P, P, LL, P, P, P, I, I, I, I, P])


class PagedKVCache:
    def __init__(self, cfg, hkv_local: int, hd: int, device):
        n, bs = cfg.num_blocks, cfg.block_size
        self.block_size = bs
        self.head_major = bool(cfg.kv_head_major)
        self.hkv, self.hd = hkv_local, hd
        shape = (n, hkv_local, bs, hd) if self.head_major else (n, bs, hkv_local, hd)
        self.k = [torch.zeros(shape, dtype=cfg.dtype, device=device) for _ in range(cfg.model.num_layers)]
        self.v = [torch.zeros(shape, dtype=cfg.dtype, device=device) for _ in range(cfg.model.num_layers)]

    def append(self, layer: int, k_src, v_src, slots):
        """k_src/v_src: [T, Hkv*D] row views (possibly strided); slots: int64 [T]."""
        kc, vc = self.k[layer], self.v[layer]
        row = self.hkv * self.hd
        if k_src.is_cuda:
            if self.head_major:
                check(native.lib().rb_kv_append_hm(native.dtype_code(kc.dtype), ptr(k_src), ptr(v_src),
                                                   k_src.stride(0), ptr(slots), ptr(kc), ptr(vc),
                                                   k_src.shape[0], self.hkv, self.hd, self.block_size,
                                                   stream_ptr()), "rb_kv_append_hm")
            else:
                check(native.lib().rb_kv_append(native.dtype_code(kc.dtype), ptr(k_src), ptr(v_src),
                                                k_src.stride(0), ptr(slots), ptr(kc), ptr(vc),
                                                k_src.shape[0], row, stream_ptr()), "rb_kv_append")
            count_launch()
        elif self.head_major:
            blk, off = slots // self.block_size, slots % self.block_size
            T = k_src.shape[0]
            kc[blk, :, off] = k_src.reshape(T, self.hkv, self.hd)
            vc[blk, :, off] = v_src.reshape(T, self.hkv, self.hd)
        else:
            kc.view(-1, row)[slots] = k_src
            vc.view(-1, row)[slots] = v_src

    def gather(self, layer: int, table: torch.Tensor, positions: torch.Tensor):
        """K and V ``[len(positions), Hkv, D]`` of logical token ``positions`` of the sequence whose
        block table is ``table``."""
        blk, off = table[positions // self.block_size], positions % self.block_size
        if self.head_major:
            return self.k[layer][blk, :, off], self.v[layer][blk, :, off]
        return self.k[layer][blk, off], self.v[layer][blk, off]


class PagedLatentCache:
    """One row per token and layer: a latent that keys and values are linear in, then the key part shared
    by all heads.  ``rows[i]`` is layer i's row width (0 or None: the layer keeps nothing, it reads the pool
    of ``share[i]``)."""

    def __init__(self, num_blocks: int, block_size: int, rows: List[int], share: List[int], dtype, device):
        self.block_size, self.share = block_size, list(share)
        self.pools: List[Optional[torch.Tensor]] = [
            torch.zeros((num_blocks, block_size, w), dtype=dtype, device=device) if w else None for w in rows]
        for i, j in enumerate(self.share):
            if self.pools[j] is None or (i != j and self.pools[i] is not None):
                raise ValueError(f"layer {i} reads the latents of layer {j}, which keeps none of its own")

    def pool(self, layer: int) -> torch.Tensor:
        """Pool ``[num_blocks, block_size, row]`` that ``layer`` attends to."""
        return self.pools[self.share[layer]]

    def owns(self, layer: int) -> bool:
        return self.pools[layer] is not None

    def bytes_per_token(self) -> int:
        return sum(p.shape[-1] * p.element_size() for p in self.pools if p is not None)


class PagedWindowCache:
    """Keys and values of layers that differ in their sizes: ``sizes[i]`` = (key/value heads, numbers per key, per
    value) of layer i, pools ``[num_blocks, heads, block_size, numbers]`` (a head's tokens of a block together); None:
    the layer keeps nothing per token.  Tokens that every window has left stay until their sequence ends."""

    def __init__(self, num_blocks: int, block_size: int, sizes: List[Optional[Tuple[int, int, int]]], dtype, device):
        self.block_size = block_size

        def pool(s, n):
            return None if s is None else torch.zeros((num_blocks, s[0], block_size, s[n]), dtype=dtype, device=device)

        self.k: List[Optional[torch.Tensor]] = [pool(s, 1) for s in sizes]
        self.v: List[Optional[torch.Tensor]] = [pool(s, 2) for s in sizes]

    def bytes_per_token(self) -> int:
        return sum(p.shape[1] * p.shape[3] * p.element_size() for p in self.k + self.v if p is not None)


class StateSlots:
    """State of a fixed size per sequence: ``layers[i]`` names layer i's tensors, (shape, type) each, and they get a
    leading dimension of ``places``, the scheduler's (a running sequence has one until it ends or is preempted).  Nothing
    is cleared in between: a portion that starts at position 0 ignores what it finds."""

    def __init__(self, places: int, layers: List[Optional[Dict[str, Tuple[tuple, torch.dtype]]]], device):
        self.device = device
        self.layers: List[Optional[Dict[str, torch.Tensor]]] = [
            None if l is None else {k: torch.zeros((places, *shape), dtype=dt, device=device) for k, (shape, dt) in l.items()}
            for l in layers]

    def __getitem__(self, layer: int) -> Dict[str, torch.Tensor]:
        return self.layers[layer]

    def bytes_per_sequence(self) -> int:
        return sum(t[0].numel() * t.element_size() for l in self.layers if l is not None for t in l.values())


class HybridCache(PagedWindowCache):
    """Pages for the layers that attend, state slots for the layers that recur; a layer may have both."""

    def __init__(self, num_blocks: int, block_size: int, sizes, places: int, states, dtype, device):
        super().__init__(num_blocks, block_size, sizes, dtype, device)
        self.state = StateSlots(places, states, device)
