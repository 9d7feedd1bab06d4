"""The Buvalix decoder: layers with a norm before and after each sub-layer over an fp32 residual stream,

    x <- x + N1b(mixer(N1(x))),     x <- x + N2b(ff(N2(x))),

and an optional range of layers that runs several times with the same weights (every pass with its own cache or state); each
pass but the first begins with x <- x + embedding output.  The norm behind a sub-layer, the addition to the stream, the
loop's addition and the norm ahead of the next sub-layer are one kernel.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..ops import api as O
from .base import Comm, ForwardBatch, GreedyTail
from .buvalix_config import BuvalixConfig, ChannelDeltaSpec
from .layered import LayeredModel
from .layers import ChannelDelta, GatedFF, GroupedAttention


class BuvalixModel(LayeredModel):
    def __init__(self, cfg: BuvalixConfig, weights: Dict[str, torch.Tensor], pool, comm: Optional[Comm] = None,
                 moe_mode: str = "ep", dtype: torch.dtype = torch.bfloat16):
        super().__init__(cfg, weights, pool, comm, moe_mode, dtype)
        self.mixers, self.ffs = [], []
        for i, l in enumerate(cfg.layers):
            m, p = l.mixer, f"l{i}.mix."
            if isinstance(m, ChannelDeltaSpec):
                self.mixers.append(ChannelDelta(weights, p, m.heads, m.kv_heads, m.dim, m.vdim, cfg.norm_eps))
            else:
                temp = (m.q_temp.coef, m.q_temp.every) if m.q_temp else None
                self.mixers.append(GroupedAttention(weights, p, m.heads, m.kv_heads, m.dim, m.vdim, m.scale, m.softcap, temp))
            self.ffs.append(None if l.ff is None else GatedFF(weights, f"l{i}.mlp.", "gelu_tanh"))

    def _norm(self, name: str):
        return self.w[name + ".w"], self.w[name + ".b"]

    def forward(self, fb: ForwardBatch, greedy: Optional[GreedyTail] = None):
        """Returns fp32 logits [n, vocab] of the rows ``fb.last_idx`` (all rows if None); with ``greedy`` returns
        (logits, greedy tokens [n] int32)."""
        cfg, eps, dt, pool = self.cfg, self.cfg.norm_eps, self.dtype, self.pool
        x, x0 = self.embed(fb, cfg.loop is not None and cfg.loop.times > 1)
        pending: dict = {}     # what the next norm has to do to the stream first
        for n, run in enumerate(self.runs):
            i = run.layer
            if run.enters:
                pending["add"] = x0
            h = O.residual_layer_norm(x, eps, dt, norm=self._norm(f"l{i}.norm1"), **pending)
            mixer = self.mixers[i]
            if isinstance(mixer, ChannelDelta):
                y = mixer(h, pool.state[n], pool.conv[n], fb)
            else:
                y = mixer(h, pool.keys[n], pool.values[n], fb)
            pending = {"sub": (y, *self._norm(f"l{i}.norm1b"))}
            if self.ffs[i] is not None:
                h = O.residual_layer_norm(x, eps, dt, norm=self._norm(f"l{i}.norm2"), **pending)
                pending = {"sub": (self.ffs[i](h), *self._norm(f"l{i}.norm2b"))}
            if self.on_run is not None:
                O.residual_layer_norm(x, eps, dt, **pending)
                pending = {}
                self.on_run(n, x)
        h = O.residual_layer_norm(x, eps, dt, norm=self._norm("final.norm"), rows=fb.last_idx, keep=False, **pending)
        return self.finish(h, self.w["head.weight"], fb, greedy)
