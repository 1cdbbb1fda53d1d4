"""Continuous-batching scheduler and paged block allocator (C++: ``csrc/serve/kv_scheduler.cpp``)."""
from __future__ import annotations

import ctypes
from ctypes import c_int, c_longlong, c_void_p
from typing import List

import torch

from ..ops import _lib


class Scheduler:
    """ctypes face of the C++ continuous-batching scheduler / block allocator."""

    def __init__(self, num_blocks: int, block_size: int, max_batch: int, token_budget: int):
        L = _lib.host_lib()
        L.rbs_create.restype = c_void_p
        L.rbs_create.argtypes = [c_int] * 4
        L.rbs_destroy.argtypes = [c_void_p]
        L.rbs_add_request.argtypes = [c_void_p, c_longlong, c_int, c_int]
        L.rbs_schedule.argtypes = [c_void_p] + [c_void_p] * 6 + [c_int]
        L.rbs_commit.argtypes = [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int, c_void_p, c_int,
                                 c_void_p, c_int]
        L.rbs_block_table.argtypes = [c_void_p, c_longlong, c_void_p, c_int]
        L.rbs_block_tables.argtypes = [c_void_p, c_void_p, c_int, c_void_p, c_int, c_void_p]
        L.rbs_places.argtypes = [c_void_p, c_void_p, c_int, c_void_p]
        L.rbs_context_len.argtypes = [c_void_p, c_longlong]
        L.rbs_abort.argtypes = [c_void_p, c_longlong]
        L.rbs_extend.argtypes = [c_void_p, c_longlong, c_int]
        for n in ("rbs_num_free_blocks", "rbs_num_waiting", "rbs_num_running"):
            getattr(L, n).argtypes = [c_void_p]
        L.rbs_num_preemptions.restype = c_longlong
        L.rbs_num_preemptions.argtypes = [c_void_p]
        self.L = L
        self.h = c_void_p(L.rbs_create(num_blocks, block_size, max_batch, token_budget))
        self.cap = max(max_batch, 64) * 4
        self.block_size = block_size

    def __del__(self):
        try:
            self.L.rbs_destroy(self.h)
        except Exception:
            pass

    def add(self, rid: int, prompt_len: int, max_new: int) -> int:
        return self.L.rbs_add_request(self.h, rid, prompt_len, max_new)

    def schedule(self):
        cap = self.cap
        dec = (c_longlong * cap)(); pre = (c_longlong * cap)()
        ps = (c_int * cap)(); pl = (c_int * cap)()
        nd, npf = c_int(0), c_int(0)
        self.L.rbs_schedule(self.h, dec, ctypes.byref(nd), pre, ps, pl, ctypes.byref(npf), cap)
        return ([dec[i] for i in range(nd.value)],
                [(pre[i], ps[i], pl[i]) for i in range(npf.value)])

    def commit(self, decode_ids, prefills, eos_ids=()):
        cap = self.cap
        dec = (c_longlong * max(1, len(decode_ids)))(*decode_ids)
        pre = (c_longlong * max(1, len(prefills)))(*[p[0] for p in prefills])
        pl = (c_int * max(1, len(prefills)))(*[p[2] for p in prefills])
        eos = (c_longlong * max(1, len(eos_ids)))(*eos_ids)
        fin = (c_longlong * cap)()
        n = self.L.rbs_commit(self.h, dec, len(decode_ids), pre, pl, len(prefills), eos, len(eos_ids),
                              fin, cap)
        return [fin[i] for i in range(n)]

    def extend(self, rid: int, n: int) -> int:
        """Makes room for the next ``n`` tokens of a caller-driven sequence (admitted at its first call) and
        returns the position of the first one; ``abort`` ends the sequence."""
        start = self.L.rbs_extend(self.h, rid, n)
        if start < 0:
            raise RuntimeError({-1: "the KV pool has too few free blocks",
                                -2: "every sequence slot is taken",
                                -3: "the id belongs to a scheduled request"}[start] + f" (sequence {rid}, {n} tokens)")
        return start

    def abort(self, rid: int) -> None:
        self.L.rbs_abort(self.h, rid)

    def block_table(self, rid: int, max_blocks: int) -> List[int]:
        out = (c_int * max_blocks)()
        n = self.L.rbs_block_table(self.h, rid, out, max_blocks)
        return [out[i] for i in range(max(0, min(n, max_blocks)))]

    def block_tables(self, rids: List[int], max_blocks: int, pin: bool = False) -> torch.Tensor:
        """Block tables of several sequences as one int32 ``[len(rids), max_blocks]`` tensor (unused
        entries zero), filled by a single native call."""
        n = len(rids)
        out = torch.empty((n, max_blocks), dtype=torch.int32, pin_memory=pin)
        counts = (c_int * n)()
        ids = (c_longlong * n)(*rids)
        missing = self.L.rbs_block_tables(self.h, ids, n, c_void_p(out.data_ptr()), max_blocks, counts)
        if missing:
            raise KeyError(f"{missing} unknown sequence id(s) in {rids}")
        return out

    def places(self, rids: List[int]) -> torch.Tensor:
        """int32 [len(rids)]: which of the ``max_batch`` places every running sequence has, from its admission until
        it ends or is preempted; models keep state of a fixed size per sequence there."""
        n = len(rids)
        out = torch.empty(n, dtype=torch.int32)
        missing = self.L.rbs_places(self.h, (c_longlong * n)(*rids), n, c_void_p(out.data_ptr()))
        if missing:
            raise KeyError(f"{missing} sequence(s) without a place in {rids}")
        return out

    def context_len(self, rid: int) -> int:
        return self.L.rbs_context_len(self.h, rid)

    def free_blocks(self) -> int:
        return self.L.rbs_num_free_blocks(self.h)

    def num_waiting(self) -> int:
        return self.L.rbs_num_waiting(self.h)

    def num_running(self) -> int:
        return self.L.rbs_num_running(self.h)

    def preemptions(self) -> int:
        return int(self.L.rbs_num_preemptions(self.h))
