"""What the layered decoders share: set-up, reports and the audit of a forward's index tensors."""
from __future__ import annotations

from typing import Callable, Dict, Optional

import torch

from ..ops import api as O
from .base import Comm, ForwardBatch


class LayeredModel:
    """Base of the layered decoders: an fp32 residual stream through ``cfg.runs``, one GPU."""

    derived_suffix = ()      # weights that repeat others in another layout (reported)

    def __init__(self, cfg, weights: Dict[str, torch.Tensor], pool, comm: Optional[Comm] = None, moe_mode: str = "ep",
                 dtype: torch.dtype = torch.bfloat16):
        self.cfg, self.w, self.pool, self.dtype = cfg, weights, pool, dtype
        self.comm = comm or Comm()
        if self.comm.size != 1:
            raise ValueError(f"the {cfg.model_type} model runs on one GPU (tensor parallel size 1)")
        self.logits_width = cfg.vocab_size
        self.runs = cfg.runs
        self.on_run: Optional[Callable[[int, torch.Tensor], None]] = None   # sees the stream after every layer run
        if weights["embed.weight"].is_cuda:
            from ..ops import native

            # weights are never written after loading: the GEMMs may fetch them ahead of the dependent-launch wait
            native.check(native.cuda_lib().dsv4_gemm_set_weight_prefetch(1), "dsv4_gemm_set_weight_prefetch")
        from ..env import ENV

        self._debug_bounds = bool(ENV.DEBUG_BOUNDS)

    def prepare_report(self) -> dict:
        by_fmt: Dict[str, int] = {}
        for v in self.w.values():
            fmt = str(v.dtype).replace("torch.", "")
            by_fmt[fmt] = by_fmt.get(fmt, 0) + v.numel() * v.element_size()
        derived = {k: v.numel() * v.element_size() for k, v in self.w.items() if k.endswith(self.derived_suffix)}
        return {"rank": 0, "world": 1, "activations": str(self.dtype).replace("torch.", ""),
                "layer_runs": len(self.runs), "bytes_by_format": by_fmt, "bytes_total": sum(by_fmt.values()),
                "derived_bytes": derived, "weight_prefetch_before_dependency_wait": self.w["embed.weight"].is_cuda}

    def audit_inputs(self, fb: ForwardBatch) -> None:
        """Checked runs (MINISGL_DEBUG_BOUNDS=1): every index tensor is audited against its range before use."""
        locs = (self.pool.sizes.num_pages + 1) * self.pool.page_size
        O.check_index(fb.input_ids, 0, self.cfg.vocab_size, "input_ids")
        O.check_index(fb.positions, 0, fb.page_table.shape[1], "positions")
        O.check_index(fb.slots, 0, fb.page_table.shape[0], "slots")
        O.check_index(fb.out_loc, -1, locs, "out_loc")
        O.check_index(fb.page_table, 0, locs, "page_table")

    def embed(self, fb: ForwardBatch, want_act: bool, **kw):
        """(fp32 stream, the embedding output as activations if wanted), with the index audit around it; kw: further arguments of
        ``embed_residual``."""
        if self._debug_bounds and fb.token_feedback is None:
            self.audit_inputs(fb)
        if "pairs" in kw:
            kw.update(positions=fb.positions, fb=fb)
        slots = fb.slots if fb.token_feedback is not None or "pairs" in kw else None
        x, x0 = O.embed_residual(fb.input_ids, self.w["embed.weight"], self.dtype, fb.token_feedback, slots, want_act, **kw)
        if self._debug_bounds and fb.token_feedback is not None:
            self.audit_inputs(fb)
        return x, x0

    def finish(self, h: torch.Tensor, head: torch.Tensor, fb: ForwardBatch, greedy):
        """fp32 logits of the normed rows; with ``greedy`` (logits, greedy tokens [n] int32)."""
        gathered = fb.last_idx is not None
        out = greedy.logits_out[: h.shape[0]] if greedy is not None and greedy.logits_out is not None else None
        logits = O.linear(h, head, out=out, out_dtype=torch.float32)
        if greedy is not None:
            slots = fb.slots[fb.last_idx] if gathered else fb.slots
            return logits, self.comm.greedy_tokens(logits, slots, None if gathered else fb.num_valid, greedy)
        return self.comm.all_gather_last(logits)
