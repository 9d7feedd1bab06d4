"""Plain-PyTorch statement of the operators of the layered models (fp32 residual stream, latent attention without
positions, recurrent time mixing, bf16 experts): the bodies CPU tensors run on.  fp32 arithmetic, results in the
activation type."""
from __future__ import annotations

import torch


def _rms(x, eps):
    return x * torch.rsqrt(x.square().mean(-1, keepdim=True) + eps)


def segments(fb):
    """Row ranges [a, b) of the requests of a forward."""
    if fb.seg_off is None:
        n = fb.positions.shape[0]
        return [(i, i + 1) for i in range(n)]
    off = fb.seg_off.tolist()
    return list(zip(off[:-1], off[1:]))


def embed_residual(ids, weight, dtype, feedback, slots, want_act, mul, table, positions, streams, pairs=None, pair_mul=(0, 0),
                   tokens=None, fb=None):
    if feedback is not None:
        ids.copy_(feedback[slots.long()])
    x = weight[ids.long()].float() * mul
    if table is not None:
        x = x + table[positions.long()].float()
    if pairs is not None:
        n, t = pairs.shape[0] - 1, ids.shape[0]
        before = [0] * t
        for i in range(t):
            p = int(positions[i])
            here = feedback is None and i and slots[i - 1] == slots[i] and int(positions[i - 1]) + 1 == p
            before[i] = int(ids[i - 1]) if here else int(tokens[fb.page_table[int(slots[i]), p - 1].long()]) if p else -1
        rows = [n if b < 0 else (b * pair_mul[0] + int(i) * pair_mul[1]) % n for b, i in zip(before, ids)]
        x = x + pairs[torch.tensor(rows)].float()
        ok = fb.out_loc >= 0
        tokens[fb.out_loc[ok].long()] = ids[ok]
    act = x.to(dtype, copy=True) if want_act else None           # the stream changes in place
    return (x if streams is None else x[:, None].repeat(1, streams, 1)), act


def stream_norm(x, eps, dtype, pre, post, sub, experts, rows, keep):
    t, s, d = x.shape
    new = x
    if post is not None:
        y = torch.zeros(t, d) if sub is None else sub
        if experts is not None:
            erows, wts, idx, n, h = experts
            real = (idx >= 0) & (idx < n)
            w = torch.where(real, wts, torch.zeros_like(wts))
            y = y + (torch.where(real[..., None], erows.float().view(*idx.shape, -1), 0.0) * w[..., None]).sum(1)
            y = y + torch.where(idx >= n, wts, torch.zeros_like(wts)).sum(1, keepdim=True) * h.float()
        new = torch.einsum("tad,ab->tbd", x, post[s:].view(s, s)) + post[:s, None] * y[:, None]
        if keep:
            x.copy_(new)
    if pre is None:
        return None
    u = torch.einsum("tsd,s->td", new if rows is None else new[rows], pre[:s])
    return (_rms(u, eps) * pre[s]).to(dtype)


def residual_norm(x, gain, eps, dtype, mul, rows, add, add2, vec, experts, cast, sub=None):
    if sub is not None:
        y, bias, sub_gain = sub
        s = _rms(y if bias is None else y + bias, eps) * sub_gain
        if rows is not None:
            x, rows = x[rows] + s[rows], None
        else:
            x += s
    for a in (add, add2, vec):
        if a is not None:
            x += a
    if experts is not None:
        erows, wts, idx = experts
        w = torch.where(idx >= 0, wts, torch.zeros_like(wts))
        x += (erows.float().view(*idx.shape, -1) * w[..., None]).sum(1)
    if gain is None:
        return x.to(dtype, copy=True) if cast else None
    y = x if rows is None else x[rows]
    return (_rms(y, eps) * gain * mul).to(dtype)


def route_topk(h, weight, bias, top, num_valid, kind, scale):
    z = h.float() @ weight.float().t()
    if kind == "selected":
        idx = torch.sort(z + bias, dim=-1, descending=True, stable=True).indices[:, :top]
        w = torch.softmax(torch.gather(z + bias, 1, idx), -1) * scale
    else:
        p = torch.softmax(z, -1)
        idx = torch.sort(p + bias, dim=-1, descending=True, stable=True).indices[:, :top]
        w = torch.gather(p, 1, idx) * scale
    idx = idx.to(torch.int32)
    if num_valid is not None:
        idx[int(num_valid):] = -1
        w[int(num_valid):] = 0
    return idx, w


def gated_experts(h, idx, wts, w13, w2):
    t, k = idx.shape
    out = torch.zeros(t, k, h.shape[1], dtype=h.dtype)
    for e in range(w13.shape[0]):
        at = (idx == e).nonzero()
        if len(at) == 0:
            continue
        x = h[at[:, 0]].float()
        g, u = x @ w13[e, 0].float().t(), x @ w13[e, 1].float().t()
        act = (g * torch.sigmoid(g) * u).to(h.dtype).float()
        out[at[:, 0], at[:, 1]] = (act @ w2[e].float().t()).to(h.dtype)
    return out.view(t * k, -1)


def latent_store(x, gain, eps, cache, fb):
    ok = fb.out_loc >= 0
    cache[fb.out_loc[ok].long()] = (_rms(x[ok].float(), eps) * gain).to(cache.dtype)


def latent_rotate_store(p, at_rot, at_c, gain, eps, freq, mul, cache, fb, heads, dim, whole):
    t, rank, rot = p.shape[0], gain.shape[0], 2 * freq.shape[0]
    a = fb.positions.float()[:, None, None] * freq
    c, s = torch.cos(a) * mul, torch.sin(a) * mul

    def turn(x):
        x = x.float().reshape(t, -1, rot)
        u, w = x[..., 0::2], x[..., 1::2]
        return torch.stack([u * c - w * s, w * c + u * s], -1).reshape(t, -1)

    lat = _rms(p[:, at_c:at_c + rank].float(), eps) * gain
    ok = fb.out_loc >= 0
    cache[fb.out_loc[ok].long()] = torch.cat([lat, turn(p[:, at_c + rank:at_c + rank + rot])], 1)[ok].to(cache.dtype)
    q = turn(p[:, at_rot:at_rot + heads * rot]).to(p.dtype)
    if not whole:
        p[:, at_rot:at_rot + heads * rot] = q
        return None
    return torch.cat([p[:, :heads * dim].reshape(t, heads, dim), q.view(t, heads, rot)], -1).reshape(t, -1)


def _hidden(fb, a, b, n, window):
    """[b - a, n]: the keys 0 .. n - 1 that the rows a .. b - 1 do not see."""
    away = fb.positions[a:b].long()[:, None] - torch.arange(n)[None, :]
    return (away < 0) | (away >= window) if window else away < 0


def latent_attention(q, cache, fb, scale, q_rot, window):
    out = torch.empty_like(q)
    heads, rank = q.shape[1:]
    for a, b in segments(fb):
        n = int(fb.positions[b - 1]) + 1
        c = cache[fb.page_table[int(fb.slots[a]), :n].long()].float()
        s = torch.einsum("thr,jr->thj", q[a:b].float(), c[:, :rank])
        if q_rot is not None:
            s = s + torch.einsum("thr,jr->thj", q_rot[a:b].float().reshape(b - a, heads, -1), c[:, rank:])
        p = torch.softmax((s * scale).masked_fill(_hidden(fb, a, b, n, window)[:, None, :], float("-inf")), -1)
        out[a:b] = torch.einsum("thj,jr->thr", p, c[:, :rank]).to(q.dtype)
    return out


def prefers_expanded(q_dtype, fb, heads, dim, vdim, rank, rot, window):
    return False


def expanded_attention(q, cache, fb, uk, uv, heads, scale, window):
    t, vdim = q.shape[0], uv.shape[0] // heads
    out = torch.empty(t, heads * vdim, dtype=q.dtype)
    for a, b in segments(fb):
        n = int(fb.positions[b - 1]) + 1
        c = cache[fb.page_table[int(fb.slots[a]), :n].long()].float()
        k, v = (c @ uk.float().t()).view(n, heads, -1), (c[:, :uv.shape[1]] @ uv.float().t()).view(n, heads, vdim)
        s = torch.einsum("thd,jhd->thj", q[a:b].float().reshape(b - a, heads, -1), k) * scale
        p = torch.softmax(s.masked_fill(_hidden(fb, a, b, n, window)[:, None, :], float("-inf")), -1)
        out[a:b] = torch.einsum("thj,jhd->thd", p, v).reshape(b - a, -1).to(q.dtype)
    return out


def mingru(p, at_u, at_g, bias_z, bias_u, state, fb, dtype):
    w = state.shape[1]
    z, u, g = p[:, :w] + bias_z, p[:, at_u:at_u + w] + bias_u, p[:, at_g:at_g + w]
    keep, b = torch.sigmoid(-z), torch.sigmoid(z) * torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    y = torch.empty(p.shape[0], w)
    for lo, hi in segments(fb):
        slot = int(fb.slots[lo])
        s = torch.zeros(w) if int(fb.positions[lo]) == 0 else state[slot].clone()
        for i in range(lo, hi):
            s = keep[i] * s + b[i]
            y[i] = s
        state[slot] = s
    return (y * g * torch.sigmoid(g)).to(dtype)


def shift_mix(x, gain, eps, mu, prev, tail, fb, dtype):
    h = _rms(x, eps) * gain
    hp = torch.cat([h[:1], h[:-1]], 0)
    for a, b in segments(fb):
        s = int(fb.slots[a])
        hp[a] = 0 if int(fb.positions[a]) == 0 else prev[s]
        (prev if b - a == 1 else tail)[s] = h[b - 1]
    return torch.cat([h + (hp - h) * m for m in mu], -1).to(dtype)


def wkv(p, a, w0, u, gain, state, prev, tail, fb, heads, eps):
    t, hd = a.shape
    d = hd // heads
    r, k, v, g = (c.view(t, heads, d) for c in p.float().chunk(4, -1))
    w = torch.exp(-torch.exp(a + w0)).view(t, heads, d)
    o = torch.empty(t, heads, d)
    for lo, hi in segments(fb):
        slot = int(fb.slots[lo])
        s = torch.zeros_like(state[slot]) if int(fb.positions[lo]) == 0 else state[slot].clone()
        for i in range(lo, hi):
            kv = k[i][:, :, None] * v[i][:, None, :]
            o[i] = ((s + u.view(heads, d)[:, :, None] * kv) * r[i][:, :, None]).sum(1)
            s = w[i][:, :, None] * s + kv
        state[slot] = s
        if hi - lo > 1:
            prev[slot] = tail[slot]
    return ((_rms(o, eps) * gain.view(heads, d) * (g * torch.sigmoid(g))).view(t, hd)).to(p.dtype)
