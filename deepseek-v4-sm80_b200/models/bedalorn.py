"""The Bedalorn decoder: pre-norm layers over an fp32 residual stream, each with its own mixer and feed-forward, and an
optional range of layers that runs several times with the same weights (every pass with its own cache or state).

Before each pass of the loop   x <- W_in [x; x0] + step[pass],   x0 being the embedding output.  W_in is applied as two
products, of which the embedding's is the same for every pass and is computed once per forward.

What a sub-layer adds to the stream is added by its last projection (fp32 accumulate into x); the weighted expert sum and
the loop's additions are added by the kernel that norms the stream next.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..ops import api as O
from .base import Comm, ForwardBatch, GreedyTail
from .bedalorn_config import BedalornConfig, DenseSpec, LatentAttentionSpec
from .layered import LayeredModel
from .layers import WKV, DenseFF, ExpertsFF, LatentAttention


class BedalornModel(LayeredModel):
    derived_suffix = ("uk_t",)

    def __init__(self, cfg: BedalornConfig, weights: Dict[str, torch.Tensor], pool, comm: Optional[Comm] = None,
                 moe_mode: str = "ep", dtype: torch.dtype = torch.bfloat16):
        super().__init__(cfg, weights, pool, comm, moe_mode, dtype)
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

    def forward(self, fb: ForwardBatch, greedy: Optional[GreedyTail] = None):
        """Returns fp32 logits [n, vocab] of the rows ``fb.last_idx`` (all rows if None); with ``greedy`` returns
        (logits, greedy tokens [n] int32)."""
        cfg, w, eps, dt = self.cfg, self.w, self.cfg.norm_eps, self.dtype
        x, x0 = self.embed(fb, cfg.loop is not None)
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
        return self.finish(h, w["embed.weight"], fb, greedy)
