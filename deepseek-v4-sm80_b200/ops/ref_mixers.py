"""Plain-PyTorch statement of the operators of the designs with grouped attention and the gated delta rule: the bodies CPU
tensors run on.  fp32 arithmetic, results in the activation type."""
from __future__ import annotations

import math

import torch

from .ref_layers import _hidden, _rms, segments


def _layer_norm(x, w, b, eps):
    c = x - x.mean(-1, keepdim=True)
    return c * torch.rsqrt(c.square().mean(-1, keepdim=True) + eps) * w + b


def residual_layer_norm(x, eps, dtype, norm, sub, add, rows, keep):
    y = x if rows is None else x[rows]
    if sub is not None:
        s = sub[0] if rows is None else sub[0][rows]
        y = y + _layer_norm(s, sub[1], sub[2], eps)
    if add is not None:
        y = y + (add if rows is None else add[rows]).float()
    if keep and rows is None:
        x.copy_(y)
    return None if norm is None else _layer_norm(y, norm[0], norm[1], eps).to(dtype)


def gated_linear(h, w, act, block, limit):
    y = (h.float() @ w.float().t()).to(h.dtype).float().view(h.shape[0], -1, 2, block)
    g, u = y[:, :, 0], y[:, :, 1]
    if act == "clamp":
        g = g.clamp(max=limit)
        a, u = g * torch.sigmoid(1.702 * g), u.clamp(-limit, limit) + 1.0
    elif act == "silu":
        a = g * torch.sigmoid(g)
    else:
        assert act == "gelu_tanh"
        a = 0.5 * g * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (g + 0.044715 * g ** 3)))
    return (a * u).reshape(h.shape[0], -1).to(h.dtype)


def rotate_store(qkv, bias, freq, q_temp, keys, values, fb, heads, kv_heads, dim, vdim, gain, unit_v, eps, v_mul):
    t = qkv.shape[0]
    x = qkv.float() if bias is None else qkv.float() + bias
    q, k, v = x.split([heads * dim, kv_heads * dim, kv_heads * vdim], 1)
    if gain is not None:
        q, k = _rms(q, eps) * gain[: heads * dim], _rms(k, eps) * gain[heads * dim:]
    if unit_v:
        v = _rms(v.reshape(t, kv_heads, vdim), eps).reshape(t, -1)
    v = v * v_mul
    pos = fb.positions

    def turn(y):
        y = y.reshape(t, -1, dim)
        if freq is None:
            return y
        n = 2 * freq.shape[0]
        a = pos.float()[:, None] * freq
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, w = y[..., 0:n:2], y[..., 1:n:2]
        return torch.cat([torch.stack([u * c - w * s, w * c + u * s], -1).flatten(2), y[..., n:]], -1)

    q, k = turn(q), turn(k)
    if q_temp is not None:
        coef, every = q_temp
        q = q * (1.0 + coef * torch.log((torch.div(pos + 1, every, rounding_mode="floor") + 1).float()))[:, None, None]
    ok = fb.out_loc >= 0
    at = fb.out_loc[ok].long()
    keys[at] = k[ok].reshape(len(at), -1).to(keys.dtype)
    values[at] = v[ok].to(values.dtype)
    return q.to(qkv.dtype)


def head_store(qkv, bias, gain, eps, freq, mul, vfreq, halves, keys, values, fb, heads, kv_heads, dim, vdim):
    t, pos = qkv.shape[0], fb.positions.float()
    x = qkv.float() if bias is None else qkv.float() + bias
    q, k, v = (y.reshape(t, -1, n) for y, n in zip(x.split([heads * dim, kv_heads * dim, kv_heads * vdim], 1), (dim, dim, vdim)))
    if gain is not None:
        q, k = _rms(q, eps) * gain[0], _rms(k, eps) * gain[1]

    def turn(y, f, m):
        if f is None:
            return y
        n, a = f.shape[0], pos[:, None, None] * f
        c, s = torch.cos(a) * m, torch.sin(a) * m
        if halves:
            u, w = y[..., :n], y[..., n:2 * n]
            return torch.cat([u * c - w * s, w * c + u * s, y[..., 2 * n:]], -1)
        u, w = y[..., 0:2 * n:2], y[..., 1:2 * n:2]
        return torch.cat([torch.stack([u * c - w * s, w * c + u * s], -1).flatten(2), y[..., 2 * n:]], -1)

    q, k, v = turn(q, freq, mul), turn(k, freq, mul), turn(v, vfreq, 1.0)
    ok = fb.out_loc >= 0
    at = fb.out_loc[ok].long()
    keys[at], values[at] = k[ok].flatten(1).to(keys.dtype), v[ok].flatten(1).to(values.dtype)
    angles = None if vfreq is None else pos[:, None] * vfreq
    return q.to(qkv.dtype), None if vfreq is None else torch.stack([torch.cos(angles), torch.sin(angles)], -1)


def grouped_attention(q, keys, values, fb, kv_heads, scale, softcap, sink, rel, slope, chunk, window, wbias, turn, gate):
    t, heads, dim = q.shape
    vdim, group = values.shape[1] // kv_heads, heads // kv_heads
    out = torch.empty(t, heads, vdim, dtype=q.dtype)
    for a, b in segments(fb):
        n = int(fb.positions[b - 1]) + 1
        locs = fb.page_table[int(fb.slots[a]), :n].long()
        k = keys[locs].float().view(n, kv_heads, dim).repeat_interleave(group, 1)
        v = values[locs].float().view(n, kv_heads, vdim).repeat_interleave(group, 1)
        s = torch.einsum("thd,jhd->htj", q[a:b].float(), k) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        away = fb.positions[a:b].long()[:, None] - torch.arange(n)[None, :]
        if rel is not None:
            s = s + rel[:, away.clamp(0, rel.shape[1] - 1)]
        if slope is not None:
            s = s - slope[:, None, None] * away
        hidden = _hidden(fb, a, b, n, window)
        if chunk:
            hidden = hidden | (torch.arange(n)[None, :] < (fb.positions[a:b].long() // chunk * chunk)[:, None])
        s = s.masked_fill(hidden, float("-inf"))
        if wbias is not None:
            p = torch.sigmoid(s + wbias[:, None, None])
            out[a:b] = _finish(torch.einsum("htj,jhe->the", p, v), a, b, turn, gate).to(q.dtype)
            continue
        if sink is not None:
            s = torch.cat([s, sink[:, None, None].expand(heads, b - a, 1)], -1)
        p = torch.softmax(s, -1)[..., :n]
        out[a:b] = _finish(torch.einsum("htj,jhe->the", p, v), a, b, turn, gate).to(q.dtype)
    return out.view(t, heads * vdim)


def _finish(o, a, b, turn, gate):
    """Results [b - a, H, e] of the rows a .. b - 1, turned back and gated."""
    if turn is not None:
        u, v = o.chunk(2, -1)
        c, s = turn[a:b, None, :, 0], turn[a:b, None, :, 1]
        o = torch.cat([u * c + v * s, v * c - u * s], -1)
    return o if gate is None else o * torch.sigmoid(gate[a:b].float())[..., None]


def conv_unit(p, taps, before, fb, heads, kv_heads, dim, vdim):
    t, n = p.shape[0], taps.shape[0]
    qk, up = kv_heads * dim, -(-kv_heads * dim // 8) * 8
    raw = torch.cat([p[:, :qk], p[:, up:up + qk], p[:, 2 * up:2 * up + heads * vdim]], 1).float()
    y = torch.empty_like(raw)
    for a, b in segments(fb):
        slot = int(fb.slots[a])
        old = before[slot].float() if int(fb.positions[a]) else torch.zeros(n - 1, raw.shape[1])
        full = torch.cat([old, raw[a:b]])
        y[a:b] = sum(full[j:j + b - a] * taps[j] for j in range(n))
    y = y * torch.sigmoid(y)
    q, k, v = y.split([qk, qk, heads * vdim], 1)
    unit = lambda x: (lambda z: z * torch.rsqrt(z.square().sum(-1, keepdim=True) + 1e-6))(x.reshape(t, kv_heads, dim))
    return (unit(q) * dim ** -0.5).reshape(t, qk), unit(k).reshape(t, qk), v.to(p.dtype)


def _keep_conv_inputs(p, before, fb, heads, kv_heads, dim, vdim):
    qk, up = kv_heads * dim, -(-kv_heads * dim // 8) * 8
    for a, b in segments(fb):
        slot, n = int(fb.slots[a]), before.shape[1]
        new = torch.cat([p[a:b, :qk], p[a:b, up:up + qk], p[a:b, 2 * up:2 * up + heads * vdim]], 1)
        old = before[slot] if int(fb.positions[a]) else torch.zeros_like(before[slot])
        before[slot] = torch.cat([old, new.to(before.dtype)])[b - a:]


def delta_rule(q, k, v, rate, dt_bias, a_log, p, at_b, gate, gain, eps, state, before, fb, heads, kv_heads):
    t, e = q.shape[0], v.shape[1] // heads
    d = q.shape[1] // kv_heads
    q, k = (x.view(t, kv_heads, d).repeat_interleave(heads // kv_heads, 1) for x in (q, k))
    vf = v.float().view(t, heads, e)
    g = torch.exp(-torch.exp(a_log)[:, None] * torch.nn.functional.softplus(rate + dt_bias, threshold=1e9).view(t, heads, d))
    beta = torch.sigmoid(p[:, at_b:at_b + heads].float())
    o = torch.empty(t, heads, e)
    for a, b in segments(fb):
        slot = int(fb.slots[a])
        s = torch.zeros_like(state[slot]) if int(fb.positions[a]) == 0 else state[slot].clone()
        for i in range(a, b):
            s = g[i][:, :, None] * s
            u = beta[i][:, None] * (vf[i] - torch.einsum("hde,hd->he", s, k[i]))
            s = s + k[i][:, :, None] * u[:, None, :]
            o[i] = torch.einsum("hde,hd->he", s, q[i])
        state[slot] = s
    _keep_conv_inputs(p, before, fb, heads, kv_heads, d, e)
    y = o * torch.rsqrt(o.square().mean(-1, keepdim=True) + eps) * gain
    return (y.reshape(t, heads * e) * torch.sigmoid(gate.float())).to(v.dtype)
