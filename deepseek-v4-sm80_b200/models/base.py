"""What every model family shares with the engine: the description of one forward, the greedy tail and the communicator
interface."""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional

import torch

from ..ops import api as O


@dataclass
class ForwardBatch:
    """Device-side description of one forward: T token rows belonging to B requests (rows of a request are consecutive
    positions and stand together)."""

    input_ids: torch.Tensor      # [T] int32
    positions: torch.Tensor      # [T] int32
    slots: torch.Tensor          # [T] int32 request table slot per row
    out_loc: torch.Tensor        # [T] int32 token location (page*page_size+offset); -1 = do not store
    last_idx: torch.Tensor       # [n] int64 rows whose logits are wanted
    page_table: torch.Tensor     # [slots+1, max_len] int32 token locations
    is_prefill: bool
    max_context: int             # max position + 1 over the batch (host value; bounds workspace widths)
    num_valid: Optional[torch.Tensor] = None  # [1] int32: rows >= num_valid are padding (graph replay)
    # [slots+1] int32 (decode only): the token of row t is token_feedback[slots[t]], the previous step's sample that
    # never left the device; the embedding kernel gathers it and fills input_ids
    token_feedback: Optional[torch.Tensor] = None
    # prefill: row ranges of the requests, request i owns rows [seg_off[i], seg_off[i+1]); decode: None, a row each
    seg_off: Optional[torch.Tensor] = None    # [B+1] int32
    seg_lens: Optional[List[int]] = None      # the same lengths on the host
    seg_ends: Optional[List[int]] = None      # context length of every request after this forward (host)
    seg_slots: Optional[List[int]] = None     # table slot of every request (host)


@dataclass
class GreedyTail:
    """Asks ``forward`` to finish with greedy sampling on the device: the argmax over the (vocabulary-parallel) logits
    is taken inside one kernel that also exchanges the shards' candidates between ranks, and the token goes to
    ``out[row]`` and to ``token_feedback[slot of the row]``.  The reference captures its greedy argmax in the decode
    graph for the same reason (python/minisgl/engine/graph.py:419-421)."""

    token_feedback: torch.Tensor   # [slots+1] int32
    out: Optional[torch.Tensor] = None  # [rows] int32 (allocated when None)
    logits_out: Optional[torch.Tensor] = None  # [rows, vocab / tp] fp32: where the head GEMM writes (else allocated)


class Comm:
    """Collectives the model needs; the single-rank default does nothing."""

    rank, size = 0, 1

    def all_reduce(self, x: torch.Tensor, tag: str = "") -> torch.Tensor:
        return x

    def all_gather_last(self, x: torch.Tensor) -> torch.Tensor:
        return x

    def greedy_tokens(self, logits_local, slots, num_valid, tail: "GreedyTail") -> torch.Tensor:
        """Greedy tokens of rows whose logits are sharded over the vocabulary; the default gathers, then picks."""
        return O.greedy_tokens(self.all_gather_last(logits_local), 0, slots, num_valid, tail.token_feedback, tail.out)
