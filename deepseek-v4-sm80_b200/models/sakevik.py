"""The Sakevik decoder: the sub-layers read the fp32 residual stream itself, and a norm stands behind each of them only,

    x <- x + N1(mixer(x)),     x <- x + N2(ff(x)).

The embedding adds a vector for the token and the one before it.  The norm behind a sub-layer (with the bias of its last projection),
the addition to the stream and the activations that the next sub-layer reads, or the norm ahead of the head, are one kernel.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..ops import api as O
from .base import Comm, ForwardBatch, GreedyTail
from .layered import LayeredModel
from .layered_config import rotary_frequencies
from .layers import GatedFF, GroupedAttention, LatentAttention, MinGRU
from .sakevik_config import MinGRUSpec, SakevikConfig, SigmoidAttentionSpec


class SakevikModel(LayeredModel):
    derived_suffix = ("uk_t",)

    def __init__(self, cfg: SakevikConfig, weights: Dict[str, torch.Tensor], pool, comm: Optional[Comm] = None,
                 moe_mode: str = "ep", dtype: torch.dtype = torch.bfloat16):
        super().__init__(cfg, weights, pool, comm, moe_mode, dtype)
        self.mixers, self.ffs = [], []
        eps = cfg.norm_eps
        for i, l in enumerate(cfg.layers):
            m, p = l.mixer, f"l{i}.mix."
            if isinstance(m, MinGRUSpec):
                self.mixers.append(MinGRU(weights, p, m.width))
            else:
                mul = rotary_frequencies(m.rot.dims, m.rot.base, m.rot.scaling)[1]
                if isinstance(m, SigmoidAttentionSpec):
                    self.mixers.append(GroupedAttention(weights, p, m.heads, m.kv_heads, m.dim, m.vdim, m.scale, eps=eps,
                                                        window=m.window, halves=True, rot_mul=mul))
                else:
                    self.mixers.append(LatentAttention(weights, p, m.heads, m.dim, m.vdim, m.kv_rank, m.scale, eps, m.rot_dim, mul,
                                                       m.window))
            self.ffs.append(None if l.ff is None else GatedFF(weights, f"l{i}.mlp.", "clamp", l.ff.limit))

    def _mix(self, n: int, h: torch.Tensor, fb: ForwardBatch) -> torch.Tensor:
        pool, mixer = self.pool, self.mixers[self.runs[n].layer]
        if isinstance(mixer, MinGRU):
            return mixer(h, pool.state[n], fb)
        if isinstance(mixer, GroupedAttention):
            return mixer(h, pool.keys[n], pool.values[n], fb)
        return mixer.mix(h, pool.latent[n], fb)

    def forward(self, fb: ForwardBatch, greedy: Optional[GreedyTail] = None):
        """Returns fp32 logits [n, vocab] of the rows ``fb.last_idx`` (all rows if None); with ``greedy`` returns
        (logits, greedy tokens [n] int32)."""
        cfg, w, eps, dt = self.cfg, self.w, self.cfg.norm_eps, self.dtype
        x, h = self.embed(fb, True, mul=cfg.embedding_scale, pairs=w["pairs.weight"],
                          pair_mul=(cfg.pairs.mul_prev, cfg.pairs.mul_cur), tokens=self.pool.tokens[0])
        sub = None                 # what the stream takes in next: (output, bias, gain of its norm)
        for n, run in enumerate(self.runs):
            l = f"l{run.layer}."
            if sub is not None:
                h = O.residual_norm(x, None, eps, dt, cast=True, sub=sub)
            sub = self._mix(n, h, fb), w.get(l + "mix.o.b"), w[l + "norm1"]
            ff = self.ffs[run.layer]
            if ff is not None:
                h = O.residual_norm(x, None, eps, dt, cast=True, sub=sub)
                sub = ff(h), None, w[l + "norm2"]
            if self.on_run is not None:
                h = O.residual_norm(x, None, eps, dt, cast=True, sub=sub)
                sub = None
                self.on_run(n, x)
        h = O.residual_norm(x, w["final.gain"], eps, dt, mul=cfg.logit_scale, rows=fb.last_idx, sub=sub)
        return self.finish(h, w["head.weight"], fb, greedy)
