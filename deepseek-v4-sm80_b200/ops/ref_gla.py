"""Plain-PyTorch statement of the operators of gated linear attention: the bodies CPU tensors run on.  fp32 arithmetic, results in
the activation type."""
from __future__ import annotations

import torch
from torch.nn.functional import logsigmoid, softplus

from .ref_layers import _rms, segments


def mlstm_gates(z, bias, cap, top, fb):
    h = top.shape[1]
    g = cap * torch.tanh((z + bias) / cap)
    i, f = g[:, :h], logsigmoid(g[:, h:])
    log_g, m = torch.empty_like(i), torch.empty_like(i)
    for a, b in segments(fb):
        slot = int(fb.slots[a])
        now = torch.zeros(h) if int(fb.positions[a]) == 0 else top[slot].clone()
        for t in range(a, b):
            m[t] = torch.maximum(f[t] + now, i[t])
            log_g[t] = f[t] + now - m[t]
            now = m[t]
        top[slot] = now
    return log_g, torch.exp(i - m), torch.exp(-m)


def causal_conv(p, taps, bias, before, fb):
    n = taps.shape[0]
    y = torch.empty(p.shape[0], p.shape[1])
    for a, b in segments(fb):
        slot = int(fb.slots[a])
        old = before[slot] if int(fb.positions[a]) else torch.zeros_like(before[slot])
        full = torch.cat([old, p[a:b].to(before.dtype)])
        y[a:b] = bias + sum(full[j:j + b - a].float() * taps[j] for j in range(n))
        before[slot] = full[b - a:]
    return (y * torch.sigmoid(y)).to(p.dtype)


def gla(kind, q, k, v, gates, state, fb, heads, groups, q_mul):
    t, (d, ew) = v.shape[0], state.shape[2:]
    e = v.shape[1] // heads
    wide = lambda x: x.float().reshape(t, groups, d).repeat_interleave(heads // groups, 1)
    vf = torch.zeros(t, heads, ew)
    vf[..., :e] = v.float().reshape(t, heads, e)
    qf = wide(q)
    if kind == "forget":
        raw, bias, low = gates
        z = raw + bias
        kf, g = ((1.0 - low) * torch.sigmoid(-z)).view(t, heads, d), (low + (1.0 - low) * torch.sigmoid(z)).view(t, heads, d)
        qf = qf * torch.sigmoid(qf)
    else:
        if kind == "given":
            log_g, fac = gates
            vf[..., e] = 1.0
        else:
            fac = softplus(gates[0] + gates[1], threshold=1e9)
            log_g = -torch.exp(gates[2]) * fac
        kf, g = wide(k) * fac[..., None], torch.exp(log_g)[..., None].expand(t, heads, d)
    out = torch.empty(t, heads, ew)
    for a, b in segments(fb):
        slot = int(fb.slots[a])
        s = torch.zeros_like(state[slot]) if int(fb.positions[a]) == 0 else state[slot].clone()
        for i in range(a, b):
            s = g[i][:, :, None] * s + kf[i][:, :, None] * vf[i][:, None, :]
            out[i] = torch.einsum("hde,hd->he", s, qf[i] * q_mul)
        state[slot] = s
    return out


def norm_heads(o, e, gain, eps, dtype, gate, floor, mul):
    t, heads, _ = o.shape
    x = o[..., :e]
    if floor is not None:
        x = x / (torch.maximum(o[..., e].abs(), floor) + 1e-6)[..., None]
    y = _rms(x, eps) * gain.view(-1, e) * mul
    y = y.reshape(t, heads * e)
    return (y if gate is None else y * torch.sigmoid(gate.float())).to(dtype)


def norm_groups(o, skip, x, z, gain, groups, eps):
    t, heads, _ = o.shape
    e = x.shape[1] // heads
    y = (o[..., :e] + skip[:, None] * x.float().reshape(t, heads, e)).reshape(t, -1)
    zf = z.float()
    y = (y * zf * torch.sigmoid(zf)).view(t, groups, -1)
    return (_rms(y, eps).reshape(t, -1) * gain).to(x.dtype)
