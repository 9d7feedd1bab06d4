"""Layer mechanisms written against the operator facade, with their sizes and constants as parameters.  Those of the designs
without a norm behind the sub-layer add to the fp32 residual stream in place, the others return their fp32 output;
activations between the projections have the serving type (bf16 or fp32)."""
from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch

from ..ops import api as O
from .base import ForwardBatch


def padded8(sizes) -> list:
    """Column ranges of parts that stand side by side, each beginning at a multiple of eight columns."""
    at, out = 0, []
    for n in sizes:
        out.append(slice(at, at + n))
        at += -(-n // 8) * 8
    return out


class LatentAttention:
    """Causal attention over one cached latent row per token.  The per-head key up-projection is absorbed into the query and the
    value up-projection into the output, so the latents are read once for all heads; long prompt portions expand the latents to keys
    and values instead, which costs fewer operations per pair.  Without positions unless ``rot`` > 0: then every query head has ``rot``
    further values that turn by its position (``freq``, cos and sin times ``rot_mul``), and a cache row one such part that all heads
    share; ``uk`` [H * (dim + rot), rank + rot] then hands that part on to every head's expanded key.  ``window`` > 0: only so many
    positions are seen."""

    def __init__(self, w: Dict[str, torch.Tensor], prefix: str, heads: int, dim: int, vdim: int, rank: int, scale: float,
                 eps: float, rot: int = 0, rot_mul: float = 1.0, window: int = 0):
        self.heads, self.dim, self.vdim, self.rank, self.scale, self.eps = heads, dim, vdim, rank, scale, eps
        self.rot, self.rot_mul, self.window = rot, rot_mul, window
        self.qc, self.gain = w[prefix + "qc"], w[prefix + "latent.gain"]
        self.uk, self.uk_t, self.uv, self.o = (w[prefix + n] for n in ("uk", "uk_t", "uv", "o"))
        if rot:
            self.freq = w[prefix + "freq"]
            self.turned, self.down = padded8([heads * dim, heads * rot, rank + rot])[1:]

    def attend(self, h: torch.Tensor, cache: torch.Tensor, fb: ForwardBatch) -> torch.Tensor:
        """The heads' results [T, H * vdim]."""
        t, hq = h.shape[0], self.heads * self.dim
        qc = O.linear(h, self.qc)
        expand = fb.is_prefill and O.prefers_expanded(qc, fb, self.heads, self.dim, self.vdim, self.rank, self.rot, self.window)
        q, q_rot = qc[:, :hq], None
        if self.rot:
            whole = O.latent_rotate_store(qc, self.turned.start, self.down.start, self.gain, self.eps, self.freq, self.rot_mul, cache,
                                          fb, self.heads, self.dim, expand)
            q, q_rot = (whole, None) if expand else (q, qc[:, self.turned])
        else:
            O.latent_store(qc[:, hq:], self.gain, self.eps, cache, fb)
        if expand:
            return O.expanded_attention(q, cache, fb, self.uk, self.uv, self.heads, self.scale, self.window)
        q = O.grouped_linear(q, self.uk_t, self.heads).view(t, self.heads, self.rank)
        lat = O.latent_attention(q, cache, fb, self.scale, q_rot, self.window)
        return O.grouped_linear(lat.view(t, self.heads * self.rank), self.uv, self.heads)

    def __call__(self, h: torch.Tensor, x: torch.Tensor, cache: torch.Tensor, fb: ForwardBatch) -> None:
        O.linear(self.attend(h, cache, fb), self.o, out=x, accumulate=True)

    def mix(self, h: torch.Tensor, cache: torch.Tensor, fb: ForwardBatch) -> torch.Tensor:
        return O.linear(self.attend(h, cache, fb), self.o, out_dtype=torch.float32)


class MinGRU:
    """Element-wise gated recurrence whose gates read only the current token, with an output gate; the logits of its gates and
    candidates are projected to 32-bit floats, with the output gate's beside them."""

    def __init__(self, w: Dict[str, torch.Tensor], prefix: str, width: int):
        self.inp, self.bias_z, self.bias_u, self.o = (w[prefix + n] for n in ("in", "z.b", "x.b", "o"))
        self.u, self.g = padded8([width] * 3)[1:]

    def __call__(self, h: torch.Tensor, state: torch.Tensor, fb: ForwardBatch) -> torch.Tensor:
        p = O.linear(h, self.inp, out_dtype=torch.float32)
        y = O.mingru(p, self.u.start, self.g.start, self.bias_z, self.bias_u, state, fb, h.dtype)
        return O.linear(y, self.o, out_dtype=torch.float32)


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


class GroupedAttention:
    """Causal attention over paged keys and values, several query heads to a key head.  Optional parts, by the weights there
    are: projection biases (``qkv.b``), rotary positions on the leading dimensions (``freq``), a sink logit per head
    (``sink``), a bias by distance (``rel``, a table, or ``slope`` per head), norms over all rows of q and of k (``qk.norm``).
    By the arguments: a query temperature (coef, every) that grows with the position; keys seen only within the query's chunk of
    positions, or in a window before it; values divided by their root mean square per head (``unit_v``) and multiplied by ``v_mul``.

    With norms per head (``head.norm`` [2, dim]) or values that turn with their positions ahead of the cache (``vfreq``; the results
    are turned back), partners of a rotation are half of the turned dimensions apart (``halves``) or neighbours, and ``rot_mul`` is a
    factor of the keys' cos and sin.  Weights may be sigmoids of score + ``wbias`` per head instead of a softmax, and heads multiplied
    by the sigmoid of a number per token (``qkvg`` instead of ``qkv``: the projection has a column per head behind q | k | v)."""

    def __init__(self, w: Dict[str, torch.Tensor], prefix: str, heads: int, kv_heads: int, dim: int, vdim: int, scale: float,
                 softcap: float = 0.0, q_temp: Optional[Tuple[float, int]] = None, chunk: int = 0, unit_v: bool = False,
                 eps: float = 0.0, v_mul: float = 1.0, window: int = 0, halves: bool = False, rot_mul: float = 1.0):
        self.window, self.halves, self.rot_mul = window, halves, rot_mul
        self.heads, self.kv_heads, self.dim, self.vdim = heads, kv_heads, dim, vdim
        self.scale, self.softcap, self.q_temp = scale, softcap, q_temp
        self.chunk, self.unit_v, self.eps, self.v_mul = chunk, unit_v, eps, v_mul
        self.qkv, self.o = w.get(prefix + "qkv"), w[prefix + "o"]
        self.bias, self.freq, self.sink, self.rel = (w.get(prefix + n) for n in ("qkv.b", "freq", "sink", "rel"))
        self.gain, self.slope = w.get(prefix + "qk.norm"), w.get(prefix + "slope")
        self.qkvg, self.wbias, self.vfreq, self.head_gain = (w.get(prefix + n) for n in ("qkvg", "wbias", "vfreq", "head.norm"))
        self.cols = padded8([heads * dim + kv_heads * (dim + vdim), heads])

    def attend(self, qkv: torch.Tensor, keys: torch.Tensor, values: torch.Tensor, fb: ForwardBatch,
               gate: Optional[torch.Tensor] = None) -> torch.Tensor:
        """What stands between the projections: q | k | v [T, ..] -> the heads' results [T, H * vdim]."""
        if self.head_gain is not None or self.vfreq is not None:
            q, turn = O.head_store(qkv, self.bias, self.head_gain, self.eps, self.freq, self.rot_mul, self.vfreq, self.halves, keys,
                                   values, fb, self.heads, self.kv_heads, self.dim, self.vdim)
            return O.grouped_attention(q, keys, values, fb, self.kv_heads, self.scale, self.softcap, self.sink, self.rel, self.slope,
                                       self.chunk, self.window, self.wbias, turn, gate)
        q = O.rotate_store(qkv, self.bias, self.freq, self.q_temp, keys, values, fb, self.heads, self.kv_heads, self.dim,
                           self.vdim, self.gain, self.unit_v, self.eps, self.v_mul)
        return O.grouped_attention(q, keys, values, fb, self.kv_heads, self.scale, self.softcap, self.sink, self.rel,
                                   self.slope, self.chunk, self.window, self.wbias, None, gate)

    def __call__(self, h: torch.Tensor, keys: torch.Tensor, values: torch.Tensor, fb: ForwardBatch) -> torch.Tensor:
        if self.qkvg is not None:
            p = O.linear(h, self.qkvg)
            qkv, gate = (p[:, c] for c in self.cols)
            return O.linear(self.attend(qkv, keys, values, fb, gate), self.o, out_dtype=torch.float32)
        return O.linear(self.attend(O.linear(h, self.qkv), keys, values, fb), self.o, out_dtype=torch.float32)


class ChannelDelta:
    """Gated delta rule with one decay per head and key channel: short convolutions over q, k and v, unit query and key
    vectors, the recurrence, per-head norm with a sigmoid gate."""

    def __init__(self, w: Dict[str, torch.Tensor], prefix: str, heads: int, kv_heads: int, dim: int, vdim: int, eps: float):
        self.heads, self.kv_heads, self.dim, self.vdim, self.eps = heads, kv_heads, dim, vdim, eps
        self.inp, self.a2, self.g2, self.o = (w[prefix + n] for n in ("in", "a2", "g2", "o"))
        self.conv, self.a_log, self.dt_bias, self.gain = (w[prefix + n] for n in ("conv", "A_log", "dt_bias", "norm"))
        up = lambda n: -(-n // 8) * 8          # every part of the merged projection starts at a multiple of eight
        ra, rg = self.a2.shape[1], self.g2.shape[1]
        qk = up(kv_heads * dim)
        self.at_v, self.at_a = 2 * qk, 2 * qk + up(heads * vdim)
        self.cols_a = slice(self.at_a, self.at_a + ra)
        self.cols_g = slice(self.at_a + up(ra), self.at_a + up(ra) + rg)
        self.at_b = self.at_a + up(ra) + up(rg)

    def __call__(self, h: torch.Tensor, state: torch.Tensor, before: torch.Tensor, fb: ForwardBatch) -> torch.Tensor:
        p = O.linear(h, self.inp)
        rate = O.linear(p[:, self.cols_a], self.a2, out_dtype=torch.float32)
        gate = O.linear(p[:, self.cols_g], self.g2)
        q, k, v = O.conv_unit(p, self.conv, before, fb, self.heads, self.kv_heads, self.dim, self.vdim)
        y = O.delta_rule(q, k, v, rate, self.dt_bias, self.a_log, p, self.at_b, gate, self.gain, self.eps, state, before, fb,
                         self.heads, self.kv_heads)
        return O.linear(y, self.o, out_dtype=torch.float32)


class GatedFF:
    """down(act(gate h) * (up h)); gate and up are one projection whose epilogue pairs them.  limit: of the gate "clamp"."""

    def __init__(self, w: Dict[str, torch.Tensor], prefix: str, act: str, limit: float = 0.0):
        self.gu, self.down, self.act, self.limit = w[prefix + "gu"], w[prefix + "down"], act, limit

    def __call__(self, h: torch.Tensor) -> torch.Tensor:
        return O.linear(O.gated_linear(h, self.gu, self.act, limit=self.limit), self.down, out_dtype=torch.float32)


class MLSTM:
    """Matrix memory with exponential input gates and a running maximum: the normaliser is one more column of the state."""

    def __init__(self, w: Dict[str, torch.Tensor], prefix: str, heads: int, dim: int, vdim: int, cap: float, eps: float):
        self.heads, self.dim, self.vdim, self.cap, self.eps = heads, dim, vdim, cap, eps
        self.inp, self.gates, self.bias, self.gain, self.o = (w[prefix + n] for n in ("in", "gates", "gates.b", "norm", "o"))
        self.cols = padded8([heads * dim, heads * dim, heads * vdim, heads * vdim])

    def __call__(self, h: torch.Tensor, state: torch.Tensor, top: torch.Tensor, fb: ForwardBatch) -> torch.Tensor:
        p = O.linear(h, self.inp)
        q, k, v, g = (p[:, c] for c in self.cols)
        log_g, fac, floor = O.mlstm_gates(O.linear(h, self.gates, out_dtype=torch.float32), self.bias, self.cap, top, fb)
        o = O.gla("given", q, k, v, (log_g, fac), state, fb, self.heads, self.heads, self.dim ** -0.5)
        y = O.norm_heads(o, self.vdim, self.gain, self.eps, h.dtype, gate=g, floor=floor)
        return O.linear(y, self.o, out_dtype=torch.float32)


class ForgetRecurrence:
    """Linear attention in which the forget gate of a key channel also decides what is written; per-head norm."""

    def __init__(self, w: Dict[str, torch.Tensor], prefix: str, heads: int, dim: int, vdim: int, eps: float, mul: float = 1.0):
        self.heads, self.dim, self.vdim, self.eps, self.mul = heads, dim, vdim, eps, mul
        self.f, self.bias, self.low, self.gain, self.o = (w[prefix + n] for n in ("f", "f.b", "lower", "norm", "o"))

    def mix(self, h: torch.Tensor, q: torch.Tensor, v: torch.Tensor, state: torch.Tensor, fb: ForwardBatch) -> torch.Tensor:
        """What stands between the projections of q and v and the output's, times ``mul``."""
        z = O.linear(h, self.f, out_dtype=torch.float32)
        o = O.gla("forget", q, None, v, (z, self.bias, self.low), state, fb, self.heads, self.heads)
        return O.norm_heads(o, self.vdim, self.gain, self.eps, h.dtype, mul=self.mul)


class ParallelMixer:
    """Attention and a recurrence side by side on the same input; their projections of it are one product (``in``)."""

    def __init__(self, w: Dict[str, torch.Tensor], prefix: str, left: GroupedAttention, right: ForgetRecurrence):
        self.inp, self.left, self.right = w[prefix + "in"], left, right
        l, r = left, right
        self.cols = padded8([l.heads * l.dim + l.kv_heads * (l.dim + l.vdim), r.heads * r.dim, r.heads * r.vdim])

    def __call__(self, h: torch.Tensor, keys: torch.Tensor, values: torch.Tensor, state: torch.Tensor,
                 fb: ForwardBatch) -> torch.Tensor:
        p = O.linear(h, self.inp)
        qkv, q, v = (p[:, c] for c in self.cols)
        y = O.linear(self.left.attend(qkv, keys, values, fb), self.left.o, out_dtype=torch.float32)
        return O.linear(self.right.mix(h, q, v, state, fb), self.right.o, out=y, accumulate=True)


class Mamba2:
    """State-space recurrence with a step size per head: one projection z | x | B | C, a short convolution over x, B and C, the
    recurrence, a skip, the gate z and norms over equal parts."""

    def __init__(self, w: Dict[str, torch.Tensor], prefix: str, heads: int, vdim: int, groups: int, state: int,
                 norm_groups: int, eps: float):
        self.heads, self.groups, self.norm_groups, self.eps = heads, groups, norm_groups, eps
        self.inp, self.dt, self.dt_bias, self.a_log = (w[prefix + n] for n in ("in", "dt", "dt_bias", "A_log"))
        self.conv, self.conv_b, self.skip, self.gain, self.o = (w[prefix + n] for n in ("conv", "conv.b", "D", "norm", "o"))
        inner, gn = heads * vdim, groups * state
        self.z, self.xbc = padded8([inner, inner + 2 * gn])
        self.x, self.b, self.c = slice(0, inner), slice(inner, inner + gn), slice(inner + gn, inner + 2 * gn)

    def __call__(self, h: torch.Tensor, state: torch.Tensor, before: torch.Tensor, fb: ForwardBatch) -> torch.Tensor:
        p = O.linear(h, self.inp)
        dt = O.linear(h, self.dt, out_dtype=torch.float32)
        u = O.causal_conv(p[:, self.xbc], self.conv, self.conv_b, before, fb)
        x = u[:, self.x]
        o = O.gla("step", u[:, self.c], u[:, self.b], x, (dt, self.dt_bias, self.a_log), state, fb, self.heads, self.groups)
        y = O.norm_groups(o, self.skip, x, p[:, self.z], self.gain, self.norm_groups, self.eps)
        return O.linear(y, self.o, out_dtype=torch.float32)


class SharedExpertsFF:
    """Mixture of silu-gated experts weighted with a softmax over all router outputs, some of which stand for the input itself,
    beside an expert that every token uses.  The weighted sum is left to the kernel that touches the streams next."""

    def __init__(self, w: Dict[str, torch.Tensor], prefix: str, top: int, scale: float):
        self.top, self.scale = top, scale
        self.router, self.bias, self.w13, self.w2 = (w[prefix + n] for n in ("router", "correction", "w13", "w2"))
        self.shared = GatedFF(w, prefix + "shared.", "silu")

    def __call__(self, h: torch.Tensor, fb: ForwardBatch) -> dict:
        idx, wts = O.route_topk(h, self.router, self.bias, self.top, fb.num_valid, "softmax", self.scale)
        rows = O.gated_experts(h, idx, wts, self.w13, self.w2)
        return {"sub": self.shared(h), "experts": (rows, wts, idx, self.w13.shape[0], h)}
