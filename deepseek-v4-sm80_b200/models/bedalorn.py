"""The Bedalorn decoder: pre-norm layers over an fp32 residual stream, each with its own mixer and feed-forward, and an
optional range of layers that runs several times with the same weights (every pass with its own cache or state).

Before each pass of the loop   x <- W_in [x; x0] + step[pass],   x0 being the embedding output.  W_in is applied as two
products, of which the embedding's is the same for every pass and is computed once per forward.

What a sub-layer adds to the stream is added by its last projection (fp32 accumulate into x); the weighted expert sum and
the loop's additions are added by the kernel that norms the stream next.
"""
from __future__ import annotations

from typing import Callable, Dict, Optional

import torch

from ..ops import api as O
from .base import Comm, ForwardBatch, GreedyTail
from .bedalorn_config import BedalornConfig, DenseSpec, LatentAttentionSpec
from .layers import WKV, DenseFF, ExpertsFF, LatentAttention


class BedalornModel:
    def __init__(self, cfg: BedalornConfig, weights: Dict[str, torch.Tensor], pool, comm: Optional[Comm] = None,
                 moe_mode: str = "ep", dtype: torch.dtype = torch.bfloat16):
        self.cfg, self.w, self.pool, self.dtype = cfg, weights, pool, dtype
        self.comm = comm or Comm()
        if self.comm.size != 1:
            raise ValueError("the Bedalorn model runs on one GPU (tensor parallel size 1)")
        self.logits_width = cfg.vocab_size
        self.runs = cfg.runs
        self.mixers, self.ffs = [], []
        eps = cfg.norm_eps
        for i, l in enumerate(cfg.layers):
            m, p = l.mixer, f"l{i}.mix."
            if isinstance(m, LatentAttentionSpec):
                self.mixers.append(LatentAttention(weights, p, m.heads, m.dim, m.vdim, m.kv_rank, m.scale, eps))
            else:
                self.mixers.append(WKV(weights, p, m.heads, m.dim, eps))
            p = f"l{i}.mlp."
            self.ffs.append(None if l.ff is None else DenseFF(weights, p) if isinstance(l.ff, DenseSpec)
                            else ExpertsFF(weights, p, l.ff.top))
        self.on_run: Optional[Callable[[int, torch.Tensor], None]] = None   # sees the stream after every layer run
        if weights["embed.weight"].is_cuda:
            from ..ops import native

            # weights are never written after loading: the GEMMs may fetch them ahead of the dependent-launch wait
            native.check(native.cuda_lib().dsv4_gemm_set_weight_prefetch(1), "dsv4_gemm_set_weight_prefetch")
        from ..env import ENV

        self._debug_bounds = bool(ENV.DEBUG_BOUNDS)

    # ------------------------------------------------------------------ reports and checks
    def prepare_report(self) -> dict:
        by_fmt: Dict[str, int] = {}
        for v in self.w.values():
            fmt = str(v.dtype).replace("torch.", "")
            by_fmt[fmt] = by_fmt.get(fmt, 0) + v.numel() * v.element_size()
        derived = {k: v.numel() * v.element_size() for k, v in self.w.items() if k.endswith("uk_t")}
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

    # ------------------------------------------------------------------ forward
    def forward(self, fb: ForwardBatch, greedy: Optional[GreedyTail] = None):
        """Returns fp32 logits [n, vocab] of the rows ``fb.last_idx`` (all rows if None); with ``greedy`` returns
        (logits, greedy tokens [n] int32)."""
        cfg, w, eps, dt = self.cfg, self.w, self.cfg.norm_eps, self.dtype
        if self._debug_bounds and fb.token_feedback is None:
            self.audit_inputs(fb)
        x, x0 = O.embed_residual(fb.input_ids, w["embed.weight"], dt, fb.token_feedback,
                                 fb.slots if fb.token_feedback is not None else None, cfg.loop is not None)
        if self._debug_bounds and fb.token_feedback is not None:
            self.audit_inputs(fb)
        pending: dict = {}     # what the next norm has to add to the stream first
        from_x0 = None
        for n, run in enumerate(self.runs):
            i = run.layer
            if run.enters is not None:
                xa = x0 if n == 0 else O.residual_norm(x, None, eps, dt, cast=True, **pending)
                if from_x0 is None:
                    from_x0 = O.linear(x0, w["loop.in_x0"], out_dtype=torch.float32)
                x = O.linear(xa, w["loop.in_x"], out_dtype=torch.float32)
                pending = {"add": from_x0, "vec": w["loop.step"][run.enters]}
            mixer, gain = self.mixers[i], w[f"l{i}.norm1.gain"]
            if isinstance(mixer, WKV):
                if pending:    # the token shift also reads the row before its own: the stream must be complete
                    O.residual_norm(x, None, eps, dt, **pending)
                    pending = {}
                mixer(x, gain, self.pool.state[n], self.pool.shift[n], self.pool.shift_tail, fb, dt)
            else:
                h = O.residual_norm(x, gain, eps, dt, **pending)
                pending = {}
                mixer(h, x, self.pool.latent[n], fb)
            if self.ffs[i] is not None:
                h = O.residual_norm(x, w[f"l{i}.norm2.gain"], eps, dt)
                pending = self.ffs[i](h, x, fb)
            if self.on_run is not None:
                if pending:
                    O.residual_norm(x, None, eps, dt, **pending)
                    pending = {}
                self.on_run(n, x)
        gathered = fb.last_idx is not None
        if gathered and pending:
            O.residual_norm(x, None, eps, dt, **pending)
            pending = {}
        h = O.residual_norm(x, w["final.gain"], eps, dt, mul=cfg.logit_scale, rows=fb.last_idx, **pending)
        out = greedy.logits_out[: h.shape[0]] if greedy is not None and greedy.logits_out is not None else None
        logits = O.linear(h, w["embed.weight"], out=out, out_dtype=torch.float32)
        if greedy is not None:
            slots = fb.slots[fb.last_idx] if gathered else fb.slots
            return logits, self.comm.greedy_tokens(logits, slots, None if gathered else fb.num_valid, greedy)
        return self.comm.all_gather_last(logits)
