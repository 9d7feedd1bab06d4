"""Storage of models whose layers keep either a paged latent row per token or a recurrent state per request.

Every *layer run* (a layer that runs several times counts each time) has its own storage:

* an attention run: ``latent[run]`` [pages * page_size, rank], one row per token, addressed by the token location
  ``page * page_size + offset``;
* a recurrent run: ``state[run]`` [slots, heads, d, d] fp32 and ``shift[run]`` [slots, width] fp32 (the last token's
  input), addressed by the request's table slot.  A slot is not cleared when it changes hands: the kernels start a
  request at position 0 from zeros.

The recurrent state of a prefix is not kept with its pages, so a model with recurrent layers does not reuse prefixes.
"""
from __future__ import annotations

from typing import Dict, Sequence, Tuple

import torch

from .paged import PagedPool, PoolSizes

# what a run keeps: ("latent", rank) or ("state", heads, d)
RunStore = Tuple


def bytes_per_page(stores: Sequence[RunStore], page_size: int, dtype: torch.dtype) -> int:
    return sum(s[1] for s in stores if s[0] == "latent") * page_size * dtype.itemsize


def bytes_per_req_slot(stores: Sequence[RunStore], width: int) -> int:
    return sum((s[1] * s[2] * s[2] + width) * 4 for s in stores if s[0] == "state")


class LatentStatePool(PagedPool):
    def __init__(self, stores: Sequence[RunStore], width: int, sizes: PoolSizes, device, dtype=torch.bfloat16):
        super().__init__(sizes, device)
        self.stores = tuple(stores)
        self.prefix_reusable = not any(s[0] == "state" for s in stores)
        rows, slots = (sizes.num_pages + 1) * sizes.page_size, sizes.num_req_slots + 1
        f32 = dict(dtype=torch.float32, device=self.device)
        self.latent: Dict[int, torch.Tensor] = {}
        self.state: Dict[int, torch.Tensor] = {}
        self.shift: Dict[int, torch.Tensor] = {}
        for run, s in enumerate(stores):
            if s[0] == "latent":
                self.latent[run] = torch.zeros(rows, s[1], dtype=dtype, device=self.device)
            else:
                self.state[run] = torch.zeros(slots, s[1], s[2], s[2], **f32)
                self.shift[run] = torch.zeros(slots, width, **f32)
        # scratch of the token shift, shared by all runs: where a portion's last row waits until the slot may change
        self.shift_tail = torch.zeros(slots, width, **f32) if self.state else None

    def storage_bytes(self) -> int:
        every = [*self.latent.values(), *self.state.values(), *self.shift.values()]
        return sum(t.numel() * t.element_size() for t in every)
