"""What serving models of decoders with an fp32 residual share: weights on their way into kernel layout, tables of a step,
products in the two precisions, and the gated delta rule's part of a mixer.

Every head and feed-forward width is padded to a multiple of eight with zero weights, which changes nothing and keeps
all operands 16-byte aligned.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..ops import native, recurrent
from ..ops.latent import prefill_items
from ..ops.stream import pad8, pad_heads, pad_to
from .batch import StepBatch
from .cache import HybridCache

SHORT_PORTION = 8


class Weights:
    """Fields of one sub-layer, set by its loader."""


class Step:
    """What one batch's sub-layers share."""

    def __init__(self, batch: StepBatch, cache: HybridCache, tabs):
        self.batch, self.cache, self.tabs, self.items = batch, cache, tabs, None
        if batch.segments:
            segs = [(s.row0, s.n, i, s.start) for i, s in enumerate(batch.segments)]
            self.items = torch.tensor(prefill_items(segs), dtype=torch.int32).to(cache.state.device)
        self._chunks: dict = {}

    def chunks(self, size: int) -> recurrent.Chunks:
        """The batch's long portions in chunks of ``size`` tokens."""
        if size not in self._chunks:
            self._chunks[size] = recurrent.cut([(g.row0, g.n) for g in self.batch.segments], size, self.cache.state.device)
        return self._chunks[size]

    def portions(self, chunked: bool):
        """(portions that go token by token, portions that go in chunks or None)."""
        b = self.batch
        return (b.seqs[:b.n_short], b.seqs[b.n_short:]) if chunked and b.segments else (b.seqs, None)


class DecoderServing:
    """Base of serving models that run on one GPU in bfloat16 or, with 32-bit kernels throughout, in float32.  A subclass
    sets ``name``, ``head`` and ``tiled_prompts`` (whether all its prompt kernels cover the model's sizes)."""

    tensor_parallel = False
    name = ""

    def __init__(self, cfg, device, seed: int, weights: Optional[Dict[str, torch.Tensor]]):
        m = cfg.model
        self.cfg, self.model, self.device = cfg, m, torch.device(device)
        if self.device.type != "cuda":
            raise RuntimeError(f"{self.name} is served by CUDA kernels; it has no CPU path")
        if cfg.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"{self.name} is served in bfloat16 or float32, not {cfg.dtype}")
        self.check_sizes(m)
        self.vocab_local = m.vocab_size
        self.exact = cfg.dtype == torch.float32      # 32-bit everywhere: no tensor cores
        if weights is None:
            weights = m.random_weights(seed, device=self.device)
        m.check_weights(weights)
        self.weights = weights
        self.dp = pad8(m.d_model)
        self.rotations: list = []                    # distinct rotations: (spec, frequencies, factor)

    @staticmethod
    def check_sizes(m) -> None:
        """Raises ValueError for sizes beyond the kernels' limits."""

    # ------------------------------------------------------------------ weights
    def _get(self, name: str) -> torch.Tensor:
        return self.weights[name].to(device=self.device, dtype=self.cfg.dtype)

    def _f32(self, name: str) -> torch.Tensor:
        return self.weights[name].to(device=self.device, dtype=torch.float32).contiguous()

    def _heads(self, name: str, heads: int, size: int) -> torch.Tensor:
        """A projection's rows by head, padded."""
        return pad_heads(self._get(name), heads, (size,), self.dp)

    def _head_columns(self, name: str, heads: int, size: int) -> torch.Tensor:
        """An output projection's columns by head, padded."""
        return pad_heads(self._get(name).t(), heads, (size,), self.model.d_model).t()

    def _by_head(self, t: torch.Tensor, heads: int, size: int) -> torch.Tensor:
        return pad_heads(t.view(-1, 1), heads, (size,), 1).view(-1).contiguous()

    def _rotation(self, spec) -> int:
        specs = [r[0] for r in self.rotations]
        if spec not in specs:
            freq, factor = spec.frequencies()
            self.rotations.append((spec, freq.to(self.device), factor))
            specs.append(spec)
        return specs.index(spec)

    def _delta_rows(self, s: Weights, p: str, r) -> List[torch.Tensor]:
        """Fields of a gated delta rule (``r``: its ``DeltaConfig``) that do not depend on its decays and output gate;
        its input rows [q | k | v]."""
        H, G, d, e = r.heads, r.kv_heads, pad8(r.dim), pad8(r.vdim)
        parts = (("q", G, r.dim), ("k", G, r.dim), ("v", H, r.vdim))
        s.delta = r
        s.taps = torch.cat([pad_heads(self._f32(f"{p}{k}.conv"), n, (size,), r.conv) for k, n, size in parts]).t().contiguous()
        s.decay = torch.exp(self._f32(p + "A_log"))
        s.head_norm = pad_to(self._f32(p + "norm"), e)
        s.chunked = recurrent.delta_chunks_covered(self.cfg.dtype, d, e)
        s.state = {"S": ((H, d, e), torch.float32), "conv": ((H, r.conv - 1, 2 * d + e), self.cfg.dtype)}
        return [self._heads(p + k, n, size) for k, n, size in parts]

    # ------------------------------------------------------------------ what the engine calls
    @property
    def rows_per_portion(self) -> Optional[int]:
        """Portions up to this length run token by token through the row kernels, longer ones in tiles of queries.
        None: all of them by rows (32-bit, or sizes the prompt kernels do not cover)."""
        return SHORT_PORTION if self.tiled_prompts else None

    def max_positions(self) -> int:
        return self.cfg.num_blocks * self.cfg.block_size

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        """fp32 logits of normed rows."""
        return self._mm(hidden, self.head, out_dtype=torch.float32)

    # ------------------------------------------------------------------ products
    def _mm(self, a: torch.Tensor, w: torch.Tensor, **kw) -> torch.Tensor:
        """``a @ w.T`` for a weight stored ``[out, in]``."""
        return native.gemm(a, w.t(), path=2 if self.exact else 0, **kw)

    def _out(self, a: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        return self._mm(a, w, out_dtype=torch.float32)

    def _few(self, s: Weights, h: torch.Tensor) -> torch.Tensor:
        """The numbers that drive a recurrence, in fp32."""
        if h.shape[0] <= recurrent.FEW_ROWS:
            return recurrent.few_outputs(h, s.w_few, s.b_few32)
        return self._mm(h, s.w_few, bias=s.b_few, out_dtype=torch.float32)

    def _heads_buffer(self, h: torch.Tensor, cols: int) -> torch.Tensor:
        return torch.empty((h.shape[0], cols), dtype=h.dtype, device=self.device)

    def _delta(self, s: Weights, st: Step, cache_id: int, raw: torch.Tensor, step: torch.Tensor, few: torch.Tensor, gate: torch.Tensor,
               out: torch.Tensor, **kw) -> None:
        """The delta rule of every portion, short ones token by token and long ones in chunks."""
        r = s.delta
        inputs = (raw, s.taps, step, s.dt, s.decay, few)
        rest = (st.cache.state[cache_id], gate, s.head_norm, out, r.kv_heads, r.dim, r.vdim, self.model.norm_eps)
        short, long = st.portions(s.chunked)
        recurrent.delta_rows(*inputs, short, *rest, **kw)
        if long is not None:
            recurrent.delta_chunks(*inputs, st.chunks(recurrent.DELTA_CHUNK), long, *rest, **kw)
