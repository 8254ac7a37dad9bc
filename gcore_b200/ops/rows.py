"""Rows of one serving step: portions of prompts first, then single tokens of decoding requests, all packed into one
batch.  Attention and recurrent mixers read from it which cache pages and state slots each row belongs to."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional

import torch


@dataclass
class PortionContexts:
    """What the portions of a step see under one attention window (0: everything), laid end to end: portion b's context
    runs from position ``start[b]`` (None: 0) to its last token."""
    cu: torch.Tensor                # [n_portions + 1] int32 offsets of the contexts
    start: Optional[torch.Tensor]   # [n_portions] int32
    rows: int                       # their total length
    max_before: int                 # longest stretch in front of a portion


def portion_contexts(first: List[int], lens: List[int], window: int):
    """Starts, offsets (host tensors), total length and longest stretch in front of the portions ``first .. first + len``."""
    start = [max(0, f - window + 1) if window else 0 for f in first]
    cu = torch.zeros(len(first) + 1, dtype=torch.int32)
    cu[1:] = torch.tensor([f + l - s for f, l, s in zip(first, lens, start)], dtype=torch.int32).cumsum(0)
    return torch.tensor(start, dtype=torch.int32), cu, int(cu[-1]), max((f - s for f, s in zip(first, start)), default=0)


@dataclass
class StepRows:
    tokens: torch.Tensor          # [T] int64
    pos: torch.Tensor             # [T] int32 position of every row in its sequence
    slots: torch.Tensor           # [T] int32 cache slot of every row (block * block_size + offset); < 0: inactive row
    tables: torch.Tensor          # [n_portions + n_single, max_blocks] int32 cache blocks of every request
    states: torch.Tensor          # [n_portions + n_single] int32 state slot of every request; < 0: inactive
    first_pos: torch.Tensor       # [n_portions + n_single] int32 position of the request's first row in this step
    cu: Optional[torch.Tensor]    # [n_portions + 1] int32 row offsets of the portions
    ctx: torch.Tensor             # [n_single] int32 context length including the new token; 0: inactive
    row_seq: torch.Tensor         # [T] int32 request of every row
    n_portions: int
    portion_rows: int             # rows that belong to portions; the rest are single tokens
    max_portion: int              # longest portion
    max_ctx: int                  # bound on every context length (fixes launch shapes)
    contexts: Dict[int, PortionContexts] = field(default_factory=dict)   # by window, for the windows the model uses

    @property
    def n_single(self) -> int:
        return self.tokens.numel() - self.portion_rows
