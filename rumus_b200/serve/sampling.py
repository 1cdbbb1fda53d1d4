"""Token selection on the device."""
from __future__ import annotations

from ctypes import c_int, c_longlong, c_void_p

import torch

from ..ops import native
from ..ops._lib import check, count_launch, ptr, stream_ptr

native.register_signature("rb_argmax", [c_int, c_void_p, c_longlong, c_int, c_int, c_void_p, c_void_p, c_void_p])


def greedy_sample(logits: torch.Tensor):
    """Row argmax -> (ids int64 [B], max values fp32 [B])."""
    if logits.is_cuda:
        B, V = logits.shape
        ids = torch.empty(B, dtype=torch.int64, device=logits.device)
        vals = torch.empty(B, dtype=torch.float32, device=logits.device)
        check(native.lib().rb_argmax(native.dtype_code(logits.dtype), ptr(logits), logits.stride(0), B, V,
                                     ptr(ids), ptr(vals), stream_ptr()), "rb_argmax")
        count_launch()
        return ids, vals
    vals, ids = logits.float().max(dim=-1)
    return ids, vals
