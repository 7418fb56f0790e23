"""What one step of the rollout engine runs: a flat list of token rows and where they belong."""

from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch


@dataclass
class StepBatch:
    """``kind``: "prompt" (every sequence starts at its first token), "decode" (every sequence goes on by one token)
    or "extend" (anything else: continued prompts, mixtures). Rows of a sequence are adjacent and in order."""

    kind: str
    tokens: torch.Tensor                 # int64 [T]
    seqs: torch.Tensor                   # int32 [T] cache sequence of each row
    positions: torch.Tensor              # int32 [T] position in its sequence
    slots: torch.Tensor                  # int64 [T] cache row
    max_len: int                         # longest run of rows of one sequence
    max_context: int                     # bound on position + 1 over the rows
    cu_seqlens: Optional[torch.Tensor] = None    # int32 [n + 1] row boundaries of the sequences (prompt)
    uniform: bool = False                # prompt: all sequences are max_len long
    want: Optional[torch.Tensor] = None  # int32 rows whose logits are asked for (None: all)
