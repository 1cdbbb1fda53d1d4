"""What one engine step computes: some tokens of some sequences, as one ragged batch."""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import List, Optional

import torch


@dataclass
class Portion:
    """The next tokens of one sequence: ``tokens`` stand at positions ``start ...``; ``want``: the places
    among them whose logits are asked for."""
    rid: int
    start: int
    tokens: List[int]
    want: List[int]


@dataclass
class Segment:
    """A prompt portion inside the batch: rows ``row0 .. row0 + n`` are tokens ``start .. start + n``."""
    start: int
    n: int
    row0: int


@dataclass
class StepBatch:
    """Rows ``0 .. n_rows`` are single tokens that attend through their own block table and context length
    (decoded tokens, and the tokens of portions too short for a tile of queries); the ``segments`` follow.
    Nothing a model reads on the host depends on the first kind beyond ``n_rows`` and ``max_ctx``, so a step
    without segments can be captured as a CUDA graph."""
    tokens: torch.Tensor                 # int64 [T]
    positions: torch.Tensor              # int64 [T]
    slots: torch.Tensor                  # int64 [T] cache slot of every token, -1 = keep nothing
    n_rows: int
    tables: Optional[torch.Tensor]       # int32 [n_rows, max_blocks]
    ctx: Optional[torch.Tensor]          # int32 [n_rows] keys the row sees, its own included
    max_ctx: int                         # no entry of ctx is larger
    segments: List[Segment]
    seg_tables: Optional[torch.Tensor]   # int32 [len(segments), max_blocks]
    # The portions themselves, for models with state per sequence: (first row, tokens, place of the sequence, position
    # of the first token).  The first ``n_short`` stand in the single rows, the segments follow; no tokens: padding.
    seqs: Optional[torch.Tensor] = None      # int32 [n_short + len(segments), 4]
    n_short: int = 0

    def to(self, device) -> "StepBatch":
        """The same batch with its tensors on ``device`` (through pinned memory when that is a GPU)."""
        gpu = torch.device(device).type == "cuda"

        def move(t):
            return t.pin_memory().to(device, non_blocking=True) if gpu else t.to(device)

        return replace(self, tokens=move(self.tokens), positions=move(self.positions), slots=move(self.slots),
                       tables=move(self.tables), ctx=move(self.ctx), seg_tables=move(self.seg_tables),
                       seqs=move(self.seqs))
