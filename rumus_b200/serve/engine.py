"""Continuous-batching inference engine: scheduler, paged cache, CUDA-graph decode, tensor parallelism.

The reference server (rumus-serve/src/{scheduler,gpu_worker,model}.rs) batches statically under a
deadline around a mock model.  Here:

* requests join and leave between steps (C++ scheduler + block allocator,
  ``csrc/serve/kv_scheduler.cpp``): each step decodes one token for every running sequence and
  spends the rest of the token budget on prompt chunks of waiting sequences;
* all tokens of a step are one batch (``serve/batch.py``) and run through the decoder stack together;
* which model runs follows from the configuration (``models/registry.py``): INT4 Llama
  (``serve/llama.py``), Zidalix (``serve/zidalix.py``), Nufupel (``serve/nufupel.py``), Potodra
  (``serve/potodra.py``), Lerosun (``serve/lerosun.py``).  A serving model brings its weights, its paged cache and state slots
  (``serve/cache.py``), ``forward(batch, cache, row_parallel)`` and ``logits(hidden)``;
* the partial-sum reductions of tensor-parallel models are all-reduces over the TP group (fused arena
  kernel or NCCL);
* ``Engine.feed`` runs token portions that the caller chooses through the same step.
"""
from __future__ import annotations

import os
import time
from dataclasses import dataclass, field
from typing import Dict, List, Optional

import torch
import torch.distributed as dist

from ..models.registry import architecture_of
from ..nn.quant import qmatmul_int4
from ..utils.metrics import trace_range
from .batch import Portion, Segment, StepBatch
from .cache import PagedKVCache
from .llama import Int4LlamaShard, paged_decode_attention
from .sampling import greedy_sample
from .scheduler import Scheduler


@dataclass
class ServeConfig:
    model: object                       # configuration of a registered architecture (models/registry.py)
    group_size: int = 128
    block_size: int = 64
    num_blocks: int = 4096
    max_batch: int = 64
    token_budget: int = 4096
    dtype: torch.dtype = torch.bfloat16
    scale_dtype: torch.dtype = torch.float16
    comm_mode: str = "nccl"
    # longest sequence (prompt + output) a request may have; None = what the model was made for, else the pool
    max_seq_len: Optional[int] = None
    # KV cache layout: False = [blocks, block_size, Hkv, D] (a token's heads together), True =
    # [blocks, Hkv, block_size, D] (a head's tokens together: long contiguous reads in decode
    # attention).  Opt-in until measured on hardware.
    kv_head_major: bool = field(default_factory=lambda: os.environ.get("RB_KV_HEAD_MAJOR", "0") == "1")
    # Decode batches run as captured CUDA graphs (one per padded batch size and context bucket): a decode
    # step is ~450 small launches whose host cost exceeds their device time.  RB_SERVE_GRAPHS=0 disables.
    cuda_graphs: bool = field(default_factory=lambda: os.environ.get("RB_SERVE_GRAPHS", "1") == "1")


@dataclass
class Request:
    rid: int
    prompt: List[int]
    max_new: int
    arrival: float = 0.0
    first_token_time: Optional[float] = None
    finish_time: Optional[float] = None
    output: List[int] = field(default_factory=list)


class Engine:
    # partial sums up to this size take the one-shot all-reduce (every rank reads all partials:
    # one flag round, latency bound); larger ones (long prompt chunks) are bandwidth bound and go
    # through NCCL's reduce-scatter / all-gather schedule
    ONESHOT_MAX_BYTES = 2 << 20
    # decode batches are padded to one of these sizes before they are captured / replayed
    GRAPH_BATCHES = (1, 2, 4, 8, 16, 24, 32, 48, 64, 96, 128, 192, 256)

    def __init__(self, cfg: ServeConfig, device=None, group: Optional[dist.ProcessGroup] = None, seed: int = 0,
                 weights: Optional[Dict[str, torch.Tensor]] = None):
        self.cfg = cfg
        self.group = group
        self.world = dist.get_world_size(group) if dist.is_initialized() else 1
        self.rank = dist.get_rank(group) if dist.is_initialized() else 0
        self.device = device or torch.device("cpu")
        model_cls = architecture_of(cfg.model).serving_class()
        if self.world > 1 and not model_cls.tensor_parallel:
            raise ValueError(f"{model_cls.__name__} runs on one rank; tensor parallelism has {self.world}")
        self.model = model_cls(cfg, self.device, self.rank, self.world, seed, weights=weights)
        self.cache = self.model.make_cache()
        self.sched = Scheduler(cfg.num_blocks, cfg.block_size, cfg.max_batch, cfg.token_budget)
        self.requests: Dict[int, Request] = {}
        self.max_seq_len = cfg.max_seq_len or self.model.max_positions()
        self.max_blocks = (self.max_seq_len + cfg.block_size - 1) // cfg.block_size
        self.steps = 0
        self.tokens_out = 0
        self._ar = None
        self._graphs: Dict[tuple, object] = {}
        self._graph_pool = None
        self._capturing = False
        self._cap_k = 0
        self.graph_replays = 0
        if self.world > 1 and cfg.comm_mode == "fused" and self.device.type == "cuda":
            from ..parallel.symm import SymmArena
            n = cfg.token_budget * cfg.model.d_model
            esz = torch.empty((), dtype=cfg.dtype).element_size()
            self.arena = SymmArena(2 * n * esz + (1 << 20), group)
            # two partial-sum buffers used in turn (see csrc/comm/oneshot_allreduce.cu)
            self._ar_bufs = [self.arena.alloc(n, cfg.dtype)[0] for _ in range(2)]
            self._ar_flags = self.arena.alloc_flags(self.world)
            self._ar_epoch = 0
            # added on the device to the epochs of captured all-reduce launches (see _decode_graph)
            self._ar_gen = torch.zeros(1, dtype=torch.int32, device=self.device)
            self.arena.barrier()
            self._ar = True

    # ------------------------------------------------------------------ requests
    def add_request(self, rid: int, prompt: List[int], max_new: int, arrival: Optional[float] = None) -> bool:
        if len(prompt) + max_new > self.max_seq_len or self.sched.add(rid, len(prompt), max_new) != 0:
            return False
        self.requests[rid] = Request(rid, list(prompt), max_new, arrival if arrival is not None else time.time())
        return True

    def has_work(self) -> bool:
        return self.sched.num_waiting() + self.sched.num_running() > 0

    # ------------------------------------------------------------------ row-parallel layer + all-reduce
    def _row_parallel(self, h: torch.Tensor, qw, residual: torch.Tensor) -> torch.Tensor:
        """``residual + sum over ranks of (h @ dequant(qw))``.  Fused mode: the matmul writes its
        partial result straight into a peer-visible buffer and ONE kernel does the flag round, the
        reduction over all ranks' partials and the residual add; NCCL mode: matmul, all-reduce, add."""
        if self.world == 1:
            return residual + qmatmul_int4(h, qw)
        if self._ar and h.shape[0] * qw.n * h.element_size() <= self.ONESHOT_MAX_BYTES:
            from ..ops.quant_cuda import int4_matmul
            from ..parallel import fused_ops
            T = h.shape[0]
            if self._capturing:
                # a captured launch keeps its arguments: its epoch is (device word) + k, k = its position in
                # the graph; the word is even at every replay, so buffer k & 1 matches the eager convention
                self._cap_k += 1
                epoch, base = self._cap_k, self._ar_gen
            else:
                self._ar_epoch += 1
                epoch, base = self._ar_epoch, None
            part = self._ar_bufs[epoch & 1][: T * qw.n].view(T, qw.n)
            int4_matmul(h, qw, out=part)
            out = torch.empty_like(residual)
            with trace_range("serve.oneshot_allreduce"):
                fused_ops.oneshot_allreduce(self.arena, part, out, flags_off=self._ar_flags,
                                            epoch=epoch, residual=residual.contiguous(), epoch_base=base)
            return out
        part = qmatmul_int4(h, qw)
        dist.all_reduce(part, group=self.group)
        return residual + part

    # ------------------------------------------------------------------ one batch
    def _make_batch(self, portions: List[Portion]):
        """The step's batch on the host (pinned on GPU engines), and the row of every wanted token in the order of
        ``portions``."""
        bs, limit = self.cfg.block_size, self.model.rows_per_portion
        lens = [len(p.tokens) for p in portions]
        order = sorted(range(len(portions)), key=lambda i: limit is not None and lens[i] > limit)   # stable
        short = [i for i in order if limit is None or lens[i] <= limit]
        n_rows = sum(lens[i] for i in short)
        tables = self.sched.block_tables([portions[i].rid for i in order], self.max_blocks)
        n = torch.tensor([lens[i] for i in order])
        start = torch.tensor([portions[i].start for i in order])
        first = torch.cumsum(n, 0) - n
        of = torch.repeat_interleave(torch.arange(len(order)), n)
        pos = start[of] + torch.arange(of.shape[0]) - first[of]
        slots = tables[of, pos // bs].long() * bs + pos % bs
        row0 = dict(zip(order, first.tolist()))
        tokens = torch.tensor([t for i in order for t in portions[i].tokens], dtype=torch.int64)
        segments = [Segment(portions[i].start, lens[i], row0[i]) for i in order[len(short):]]
        ctx = (pos[:n_rows] + 1).to(torch.int32)
        seqs = torch.stack([first.int(), n.int(), self.sched.places([portions[i].rid for i in order]), start.int()], 1)
        batch = StepBatch(tokens, pos, slots, n_rows, tables[of[:n_rows]], ctx, int(ctx.max()) if n_rows else 0, segments,
                          tables[len(short):], seqs, len(short))
        return batch, [row0[i] + w for i, p in enumerate(portions) for w in p.want]

    def _run(self, portions: List[Portion]) -> Optional[torch.Tensor]:
        """Computes one batch; returns the logits (this rank's part of the vocabulary) of the wanted tokens in
        the order of ``portions``, or None when none are wanted."""
        batch, rows = self._make_batch(portions)
        hidden = None
        with trace_range("serve.batch"):
            if not batch.segments and self.cfg.cuda_graphs and self.device.type == "cuda":
                hidden = self._decode_graph(batch)
            if hidden is None:
                hidden = self.model.forward(batch.to(self.device), self.cache, self._row_parallel)
        if not rows:
            return None
        if rows != list(range(hidden.shape[0])):
            hidden = hidden.index_select(0, torch.tensor(rows, dtype=torch.int64, device=self.device))
        return self.model.logits(hidden)

    def _argmax(self, logits: torch.Tensor) -> torch.Tensor:
        ids, vals = greedy_sample(logits)
        if self.world == 1:
            return ids
        ids = ids + self.rank * self.model.vocab_local
        allv = [torch.empty_like(vals) for _ in range(self.world)]
        alli = [torch.empty_like(ids) for _ in range(self.world)]
        dist.all_gather(allv, vals, group=self.group)
        dist.all_gather(alli, ids, group=self.group)
        best = torch.stack(allv).argmax(dim=0)
        return torch.stack(alli).gather(0, best[None]).squeeze(0)

    # ------------------------------------------------------------------ caller-driven sequences
    def feed(self, portions: List[tuple]) -> Optional[torch.Tensor]:
        """Runs the next tokens of several sequences as one batch, from the cache that earlier calls left:
        ``portions`` holds ``(id, tokens, wanted places)`` and the logits of the wanted places come back as one
        ``[n, vocab]`` tensor in that order (None if there are none).  A sequence is admitted at its first
        portion and lives until ``release``; the scheduler's own requests are left alone."""
        todo = []
        for rid, tokens, want in portions:
            todo.append(Portion(rid, self.sched.extend(rid, len(tokens)), list(tokens), list(want)))
        return self._run(todo)

    def release(self, rid: int) -> None:
        """Ends a caller-driven sequence: its cache blocks are free again."""
        self.sched.abort(rid)

    # ------------------------------------------------------------------ decode step as a CUDA graph
    def _split_rows(self, t: torch.Tensor, Bp: int):
        """Views of a graph's int32 inputs: sequences (first: they are read as groups of four), context lengths,
        block tables."""
        seqs, ctx, tables = t.split([4 * Bp, Bp, Bp * self.max_blocks])
        return seqs.view(Bp, 4), ctx, tables.view(Bp, self.max_blocks)

    def _capture_decode(self, Bp: int, ctx_bucket: int):
        """Captures the decoder stack for ``Bp`` single-token rows whose contexts fit ``ctx_bucket`` tokens.
        Inputs live in static device tensors; padded rows carry cache slot -1 (the append kernels skip them),
        context length 1, block table 0 and no sequence, and their outputs are ignored."""
        from types import SimpleNamespace
        dev = self.device
        st = SimpleNamespace(ints=torch.empty(3 * Bp, dtype=torch.int64, device=dev),
                             rows=torch.empty(Bp * (self.max_blocks + 5), dtype=torch.int32, device=dev))
        seqs, ctx, tables = self._split_rows(st.rows, Bp)
        b = StepBatch(tokens=st.ints[:Bp], positions=st.ints[Bp:2 * Bp], slots=st.ints[2 * Bp:], n_rows=Bp,
                      tables=tables, ctx=ctx, max_ctx=ctx_bucket, segments=[], seg_tables=None, seqs=seqs, n_short=Bp)
        st.batch = b
        for t, v in ((b.tokens, 0), (b.positions, 0), (b.slots, -1), (b.tables, 0), (b.ctx, 1), (b.seqs, 0)):
            t.fill_(v)

        # one eager pass first, on a side stream: whatever the kernels set up lazily (function attributes,
        # workspaces, communicator channels) exists before the capture begins
        cur = torch.cuda.current_stream(dev)
        side = torch.cuda.Stream(dev)
        side.wait_stream(cur)
        with torch.cuda.stream(side):
            self.model.forward(b, self.cache, self._row_parallel)
        cur.wait_stream(side)
        torch.cuda.synchronize(dev)
        g = torch.cuda.CUDAGraph()
        self._capturing, self._cap_k = True, 0
        try:
            with torch.cuda.graph(g, pool=self._graph_pool, capture_error_mode="thread_local"):
                st.hidden = self.model.forward(b, self.cache, self._row_parallel)
        finally:
            self._capturing = False
        if self._graph_pool is None:
            self._graph_pool = g.pool()
        st.graph, st.n_allreduce = g, self._cap_k
        return st

    def warmup_graphs(self, max_ctx: Optional[int] = None) -> int:
        """Captures the decode graphs a run can meet (every padded batch size up to ``max_batch``, every
        context bucket up to ``max_ctx``) before traffic arrives, so that no request waits for a capture.
        Every tensor-parallel rank has to call it (the captures run collectives).  Returns how many."""
        if not (self.cfg.cuda_graphs and self.device.type == "cuda"):
            return 0
        top = max_ctx or self.max_seq_len
        n, cb = 0, 256
        while True:
            for Bp in self.GRAPH_BATCHES:
                if (Bp, cb) not in self._graphs:
                    self._graphs[(Bp, cb)] = self._capture_decode(Bp, cb)
                    n += 1
                if Bp >= self.cfg.max_batch:
                    break
            if cb >= top:
                break
            cb *= 2
        return n

    def _decode_graph(self, batch: StepBatch):
        """Runs the decoder stack for a batch of single-token rows by replaying a captured graph; returns the
        hidden states ``[n_rows, d]``, or None when the batch is larger than the largest captured size."""
        B = batch.n_rows
        Bp = next((b for b in self.GRAPH_BATCHES if b >= B), None)
        if Bp is None:
            return None
        ctx_bucket = max(256, 1 << (batch.max_ctx - 1).bit_length())
        st = self._graphs.get((Bp, ctx_bucket))
        if st is None:
            st = self._graphs[(Bp, ctx_bucket)] = self._capture_decode(Bp, ctx_bucket)
        ints = torch.zeros((3, Bp), dtype=torch.int64, pin_memory=True)
        for r, v in enumerate((batch.tokens, batch.positions, batch.slots)):
            ints[r, :B] = v
        ints[2, B:] = -1
        rows = torch.zeros(Bp * (self.max_blocks + 5), dtype=torch.int32, pin_memory=True)
        seqs, ctx, tables = self._split_rows(rows, Bp)
        seqs[:batch.n_short] = batch.seqs
        ctx[:B], ctx[B:] = batch.ctx, 1
        tables[:B] = batch.tables
        st.ints.copy_(ints.view(-1), non_blocking=True)
        st.rows.copy_(rows, non_blocking=True)
        if self._ar and st.n_allreduce:
            if self._ar_epoch & 1:
                self._ar_epoch += 1          # every rank skips the same epoch number; flags only ever grow
            self._ar_gen.fill_(self._ar_epoch)
            self._ar_epoch += st.n_allreduce
        st.graph.replay()
        self.graph_replays += 1
        return st.hidden[:B]

    # ------------------------------------------------------------------ one engine step
    def step(self) -> List[int]:
        """Runs one scheduling step; returns the ids of requests that finished."""
        with trace_range("serve.schedule"):
            decode_ids, prefills = self.sched.schedule()
        if not decode_ids and not prefills:
            return []
        portions = []
        for rid in decode_ids:
            req = self.requests[rid]
            n = len(req.prompt) + len(req.output)
            portions.append(Portion(rid, n - 1, [req.output[-1] if req.output else req.prompt[-1]], [0]))
        for rid, start, n in prefills:
            req = self.requests[rid]
            seq = req.prompt + req.output   # a preempted sequence re-prefills what it had generated
            portions.append(Portion(rid, start, seq[start:start + n], [n - 1] if start + n >= len(seq) else []))
        logits = self._run(portions)
        t_now = time.time()
        if logits is not None:
            ids = self._argmax(logits).tolist()
            t_now = time.time()
            for rid, tok in zip([p.rid for p in portions if p.want], ids):
                req = self.requests[rid]
                if req.first_token_time is None:
                    req.first_token_time = t_now
                req.output.append(int(tok))
                self.tokens_out += 1
        finished = self.sched.commit(decode_ids, prefills)
        for rid in finished:
            self.requests[rid].finish_time = t_now
        self.steps += 1
        return finished
