"""Rows of one serving step: portions of prompts first, then single tokens of decoding requests, all packed into one
batch.  Attention and recurrent mixers read from it which cache pages and state slots each row belongs to."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch


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
    cu_ctx: Optional[torch.Tensor] = None   # [n_portions + 1] int32 offsets of the portions' whole contexts, laid end to end
    ctx_rows: int = 0                       # their total length
    max_first: int = 0                      # longest context in front of a portion

    @property
    def n_single(self) -> int:
        return self.tokens.numel() - self.portion_rows
