"""Storage of the layered models: every *layer run* (a layer that runs several times counts each time) has its own, of one
of these kinds.

Paged, one row per token, addressed by the token location ``page * page_size + offset``:

* ("latent", rank): ``latent[run]`` [pages * page_size, rank];
* ("kv", key width, value width): ``keys[run]`` and ``values[run]`` [pages * page_size, width];
* ("tokens",): ``tokens[run]`` [pages * page_size] int32, the sequence itself (for layers that read the token before).

Per request, addressed by its table slot.  A slot is not cleared when it changes hands: the kernels start a request at
position 0 from zeros.

* ("state", heads, d): ``state[run]`` [slots, heads, d, d] fp32 and ``shift[run]`` [slots, width] fp32 (the last token's
  input);
* ("delta", heads, d, e, channels, taps): ``state[run]`` [slots, heads, d, e] fp32 and ``conv[run]`` [slots, taps - 1,
  channels], the last inputs of the short convolutions, oldest first;
* ("linear", heads, d, columns, tops, channels, taps): ``state[run]`` [slots, heads, d, columns] fp32, ``top[run]`` [slots, tops]
  fp32, running maxima, and ``conv[run]`` as above; tops or channels may be 0: then there is none;
* ("vector", width): ``state[run]`` [slots, width] fp32.

A run may keep things of several kinds, ``(kind, kind, ..)``, as long as no two have the same storage.

The recurrent state of a prefix is not kept with its pages, so a model with recurrent layers does not reuse prefixes.
"""
from __future__ import annotations

from typing import Dict, List, Sequence, Tuple

import torch

from .paged import PagedPool, PoolSizes

RunStore = Tuple      # what a run keeps, as listed above
PAGED = ("latent", "kv", "tokens")


def kinds(stores: Sequence[RunStore]):
    """(run, kind) of everything that is kept."""
    for run, s in enumerate(stores):
        for k in (s,) if isinstance(s[0], str) else s:
            yield run, k


def bytes_per_page(stores: Sequence[RunStore], page_size: int, dtype: torch.dtype) -> int:
    row = lambda s: 4 if s[0] == "tokens" else sum(s[1:]) * dtype.itemsize
    return sum(row(s) for _, s in kinds(stores) if s[0] in PAGED) * page_size


def bytes_per_req_slot(stores: Sequence[RunStore], width: int, dtype: torch.dtype) -> int:
    total = 0
    for _, s in kinds(stores):
        if s[0] == "state":
            total += (s[1] * s[2] * s[2] + width) * 4
        elif s[0] == "delta":
            total += s[1] * s[2] * s[3] * 4 + (s[5] - 1) * s[4] * dtype.itemsize
        elif s[0] == "linear":
            total += (s[1] * s[2] * s[3] + s[4]) * 4 + (s[6] - 1) * s[5] * dtype.itemsize
        elif s[0] == "vector":
            total += s[1] * 4
    return total


class LayeredPool(PagedPool):
    def __init__(self, stores: Sequence[RunStore], width: int, sizes: PoolSizes, device, dtype=torch.bfloat16):
        super().__init__(sizes, device)
        self.stores = tuple(stores)
        self.prefix_reusable = all(s[0] in PAGED for _, s in kinds(stores))
        rows, slots = (sizes.num_pages + 1) * sizes.page_size, sizes.num_req_slots + 1
        act, f32 = dict(dtype=dtype, device=self.device), dict(dtype=torch.float32, device=self.device)
        self.latent: Dict[int, torch.Tensor] = {}
        self.keys: Dict[int, torch.Tensor] = {}
        self.values: Dict[int, torch.Tensor] = {}
        self.state: Dict[int, torch.Tensor] = {}
        self.shift: Dict[int, torch.Tensor] = {}
        self.conv: Dict[int, torch.Tensor] = {}
        self.top: Dict[int, torch.Tensor] = {}
        self.tokens: Dict[int, torch.Tensor] = {}
        for run, s in kinds(stores):
            if s[0] == "latent":
                self.latent[run] = torch.zeros(rows, s[1], **act)
            elif s[0] == "kv":
                self.keys[run], self.values[run] = torch.zeros(rows, s[1], **act), torch.zeros(rows, s[2], **act)
            elif s[0] == "tokens":
                self.tokens[run] = torch.zeros(rows, dtype=torch.int32, device=self.device)
            elif s[0] == "vector":
                self.state[run] = torch.zeros(slots, s[1], **f32)
            elif s[0] == "state":
                self.state[run] = torch.zeros(slots, s[1], s[2], s[2], **f32)
                self.shift[run] = torch.zeros(slots, width, **f32)
            elif s[0] == "delta":
                self.state[run] = torch.zeros(slots, s[1], s[2], s[3], **f32)
                self.conv[run] = torch.zeros(slots, s[5] - 1, s[4], **act)
            elif s[0] == "linear":
                self.state[run] = torch.zeros(slots, s[1], s[2], s[3], **f32)
                if s[4]:
                    self.top[run] = torch.zeros(slots, s[4], **f32)
                if s[5]:
                    self.conv[run] = torch.zeros(slots, s[6] - 1, s[5], **act)
            else:
                raise ValueError(f"unknown kind of storage {s[0]!r}")
        # scratch of the token shift, shared by all runs: where a portion's last row waits until the slot may change
        self.shift_tail = torch.zeros(slots, width, **f32) if self.shift else None

    def storage(self) -> List[torch.Tensor]:
        all_kinds = (self.latent, self.keys, self.values, self.state, self.shift, self.conv, self.top, self.tokens)
        return [t for kind in all_kinds for t in kind.values()]

    def storage_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self.storage())
