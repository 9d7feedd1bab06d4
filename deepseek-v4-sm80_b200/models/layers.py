"""Layer mechanisms written against the operator facade, with their sizes and constants as parameters.  They read an fp32
residual stream and add to it in place; activations between the projections have the serving type (bf16 or fp32)."""
from __future__ import annotations

from typing import Dict

import torch

from ..ops import api as O
from .base import ForwardBatch


class LatentAttention:
    """Causal attention without positions over one cached latent row per token.  The per-head key up-projection is
    absorbed into the query and the value up-projection into the output, so the latents are read once for all heads; long
    prompt portions expand the latents to keys and values instead, which costs fewer operations per pair."""

    def __init__(self, w: Dict[str, torch.Tensor], prefix: str, heads: int, dim: int, vdim: int, rank: int, scale: float,
                 eps: float):
        self.heads, self.dim, self.vdim, self.rank, self.scale, self.eps = heads, dim, vdim, rank, scale, eps
        self.qc, self.gain = w[prefix + "qc"], w[prefix + "latent.gain"]
        self.uk, self.uk_t, self.uv, self.o = (w[prefix + n] for n in ("uk", "uk_t", "uv", "o"))

    def __call__(self, h: torch.Tensor, x: torch.Tensor, cache: torch.Tensor, fb: ForwardBatch) -> None:
        t, hq = h.shape[0], self.heads * self.dim
        qc = O.linear(h, self.qc)
        O.latent_store(qc[:, hq:], self.gain, self.eps, cache, fb)
        if fb.is_prefill and O.prefers_expanded(qc, fb, self.heads, self.dim, self.vdim, self.rank):
            v = O.expanded_attention(qc[:, :hq], cache, fb, self.uk, self.uv, self.heads, self.scale)
        else:
            q = O.grouped_linear(qc[:, :hq], self.uk_t, self.heads).view(t, self.heads, self.rank)
            lat = O.latent_attention(q, cache, fb, self.scale)
            v = O.grouped_linear(lat.view(t, self.heads * self.rank), self.uv, self.heads)
        O.linear(v, self.o, out=x, accumulate=True)


class WKV:
    """Recurrent time mixing: token shift with five learned mixes, per-channel decays through a low-rank projection, the
    recurrence with its current-token bonus, per-head norm and gate."""

    def __init__(self, w: Dict[str, torch.Tensor], prefix: str, heads: int, dim: int, eps: float):
        self.heads, self.dim, self.eps = heads, dim, eps
        self.mu, self.rkvg, self.w1, self.w2 = (w[prefix + n] for n in ("mu", "rkvg", "w1", "w2"))
        self.w0, self.u, self.gain, self.o = (w[prefix + n] for n in ("w0", "u", "out.gain", "o"))

    def __call__(self, x: torch.Tensor, norm_gain: torch.Tensor, state, shift, tail, fb: ForwardBatch, dtype) -> None:
        d = x.shape[1]
        mixed = O.shift_mix(x, norm_gain, self.eps, self.mu, shift, tail, fb, dtype)
        p = O.grouped_linear(mixed[:, : 4 * d], self.rkvg, 4)
        low = O.linear(mixed[:, 4 * d:], self.w1, act="tanh")
        a = O.linear(low, self.w2, out_dtype=torch.float32)
        y = O.wkv(p, a, self.w0, self.u, self.gain, state, shift, tail, fb, self.heads, self.eps)
        O.linear(y, self.o, out=x, accumulate=True)


class DenseFF:
    """down(relu(up h)^2), added to the stream by the second projection."""

    def __init__(self, w: Dict[str, torch.Tensor], prefix: str):
        self.up, self.down = w[prefix + "up"], w[prefix + "down"]

    def __call__(self, h: torch.Tensor, x: torch.Tensor, fb: ForwardBatch) -> dict:
        O.linear(O.linear(h, self.up, act="relu2"), self.down, out=x, accumulate=True)
        return {}


class ExpertsFF:
    """Mixture of silu-gated experts weighted with the softmax over the chosen logits.  The weighted sum is left to the
    next kernel that touches the stream: what it has to add is returned."""

    def __init__(self, w: Dict[str, torch.Tensor], prefix: str, top: int):
        self.top = top
        self.router, self.bias, self.w13, self.w2 = (w[prefix + n] for n in ("router", "router.b", "w13", "w2"))

    def __call__(self, h: torch.Tensor, x: torch.Tensor, fb: ForwardBatch) -> dict:
        idx, wts = O.route_topk(h, self.router, self.bias, self.top, fb.num_valid)
        return {"experts": (O.gated_experts(h, idx, wts, self.w13, self.w2), wts, idx)}
