"""The Zazilix decoder: pre-norm layers over several fp32 residual streams with constant mixing weights.  A sub-layer reads a
weighted sum of the streams; its output goes back into all of them while they mix,

    h = N(sum_s in[s] x_s),    x_t <- sum_s mix[s, t] x_s + out[t] f(h),

and ahead of the head the streams are added up.  The update behind a sub-layer (with the weighted sum over its experts, where it
has some), the sum ahead of the next one and that one's norm are one kernel.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..ops import api as O
from .base import Comm, ForwardBatch, GreedyTail
from .layered import LayeredModel
from .layers import MLSTM, ForgetRecurrence, GroupedAttention, Mamba2, ParallelMixer, SharedExpertsFF
from .zazilix_config import MLSTMSpec, ParallelSpec, ZazilixConfig


class ZazilixModel(LayeredModel):
    def __init__(self, cfg: ZazilixConfig, weights: Dict[str, torch.Tensor], pool, comm: Optional[Comm] = None,
                 moe_mode: str = "ep", dtype: torch.dtype = torch.bfloat16):
        super().__init__(cfg, weights, pool, comm, moe_mode, dtype)
        self.mixers, self.ffs = [], []
        eps = cfg.norm_eps
        for i, l in enumerate(cfg.layers):
            m, p = l.mixer, f"l{i}.mix."
            if isinstance(m, MLSTMSpec):
                self.mixers.append(MLSTM(weights, p, m.heads, m.dim, m.vdim, m.gate_cap, eps))
            elif isinstance(m, ParallelSpec):
                a, r = m.left, m.right
                left = GroupedAttention(weights, p + "left.", a.heads, a.kv_heads, a.dim, a.vdim, a.scale, chunk=a.chunk,
                                        unit_v=True, eps=eps, v_mul=m.left_scale)
                right = ForgetRecurrence(weights, p + "right.", r.heads, r.dim, r.vdim, eps, m.right_scale)
                self.mixers.append(ParallelMixer(weights, p, left, right))
            else:
                self.mixers.append(Mamba2(weights, p, m.heads, m.vdim, m.groups, m.state, m.norm_groups, eps))
            self.ffs.append(None if l.ff is None else SharedExpertsFF(weights, f"l{i}.mlp.", l.ff.top, l.ff.scale))

    def _mix(self, n: int, h: torch.Tensor, fb: ForwardBatch) -> torch.Tensor:
        pool, mixer = self.pool, self.mixers[self.runs[n].layer]
        if isinstance(mixer, MLSTM):
            return mixer(h, pool.state[n], pool.top[n], fb)
        if isinstance(mixer, ParallelMixer):
            return mixer(h, pool.keys[n], pool.values[n], pool.state[n], fb)
        return mixer(h, pool.state[n], pool.conv[n], fb)

    def forward(self, fb: ForwardBatch, greedy: Optional[GreedyTail] = None):
        """Returns fp32 logits [n, vocab] of the rows ``fb.last_idx`` (all rows if None); with ``greedy`` returns
        (logits, greedy tokens [n] int32)."""
        cfg, w, eps, dt = self.cfg, self.w, self.cfg.norm_eps, self.dtype
        x, _ = self.embed(fb, False, mul=cfg.embedding_scale, table=w["pos.weight"], positions=fb.positions,
                          streams=cfg.streams)
        pending: dict = {}     # what the streams take in before the next sub-layer reads them
        for n, run in enumerate(self.runs):
            l = f"l{run.layer}."
            h = O.stream_norm(x, eps, dt, pre=w[l + "hc1.pre"], **pending)
            pending = {"post": w[l + "hc1.post"], "sub": self._mix(n, h, fb)}
            ff = self.ffs[run.layer]
            if ff is not None:
                h = O.stream_norm(x, eps, dt, pre=w[l + "hc2.pre"], **pending)
                pending = {"post": w[l + "hc2.post"], **ff(h, fb)}
            if self.on_run is not None:
                O.stream_norm(x, eps, dt, **pending)
                pending = {}
                self.on_run(n, x.sum(1))
        h = O.stream_norm(x, eps, dt, pre=w["final.pre"], rows=fb.last_idx, keep=False, **pending)
        return self.finish(h, w["head.weight"], fb, greedy)
