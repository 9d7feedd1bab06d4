"""Plain, slow statement of the Zazilix design on the CPU, in float64, one function per mechanism and one sequence at a
time.  It is written from the design's equations and shares no code with the package; the tests compare the package with
it.  Also makes small random models (configuration dict + tensors) in the checkpoint's own names and layout."""
import json
import math
import os

import torch

F = torch.float64


# ----------------------------------------------------------------------------------------------- small pieces
def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return x.clamp_min(0) + torch.log1p(torch.exp(-x.abs()))


def log_sigmoid(x):
    return -softplus(-x)


# ----------------------------------------------------------------------------------------------- streams
def stream_in(streams, weights):
    """streams [s, T, D] -> their weighted sum [T, D]."""
    return sum(w * x for w, x in zip(weights, streams))


def stream_out(streams, mix, out, y):
    """Every stream anew from all old ones (mix[from, to]) and the sub-layer's output."""
    n = streams.shape[0]
    return torch.stack([sum(mix[s, t] * streams[s] for s in range(n)) + out[t] * y for t in range(n)])


# ----------------------------------------------------------------------------------------------- mixers
def mlstm_recurrence(q, k, v, i, f, state):
    """q, k [T, H, d]; v [T, H, e]; log gates i, f [T, H]; state (S [H, d, e], n [H, d], m [H])."""
    s, n, m = state
    out = []
    for t in range(q.shape[0]):
        top = torch.maximum(f[t] + m, i[t])
        keep, write = torch.exp(f[t] + m - top), torch.exp(i[t] - top)
        s = keep[:, None, None] * s + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        m = top
        dot = (n * q[t]).sum(-1).abs()
        out.append((s * q[t][:, :, None]).sum(1) / (torch.maximum(dot, torch.exp(-m)) + 1e-6)[:, None])
    return torch.stack(out), (s, n, m)


def mlstm_mixer(h, p, m, eps, past):
    t, heads, d, e, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    if past is None:
        past = (torch.zeros(heads, d, e, dtype=F), torch.zeros(heads, d, dtype=F), torch.zeros(heads, dtype=F))
    q, k, v = (h @ p["q"].T).view(t, heads, d) / math.sqrt(d), (h @ p["k"].T).view(t, heads, d), (h @ p["v"].T).view(t, heads, e)
    capped = lambda x: cap * torch.tanh(x / cap)
    i, f = capped(h @ p["i"].T + p["i.b"]), log_sigmoid(capped(h @ p["f"].T + p["f.b"]))
    o, past = mlstm_recurrence(q, k, v, i, f, past)
    y = rms(o, eps).reshape(t, heads * e) * p["norm"] * sigmoid(h @ p["g"].T)
    return y @ p["o"].T, past


def slopes(heads):
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def chunk_attend(q, k, v, scale, size):
    """q [T, H, dim] at the last T places of k [n, G, dim], v [n, G, vdim].  Only keys of the query's own chunk of ``size``
    positions are seen; a bias falls with the distance; one is added to the sum of the weights."""
    t, heads = q.shape[:2]
    n, groups = k.shape[:2]
    out = torch.zeros(t, heads, v.shape[2], dtype=F)
    for h in range(heads):
        g, slope = h // (heads // groups), slopes(heads)[h]
        for r in range(t):
            i = n - t + r
            lo = i // size * size
            s = k[lo:i + 1, g] @ q[r, h] * scale - slope * (i - torch.arange(lo, i + 1, dtype=F))
            top = max(float(s.max()), 0.0)
            w = torch.exp(s - top)
            out[r, h] = (w / (w.sum() + math.exp(-top))) @ v[lo:i + 1, g]
    return out


def attention_mixer(h, p, m, eps, past):
    """past: None or (keys, values), both as they are cached."""
    t, heads, g = h.shape[0], m["heads"], m["kv_heads"]
    q = (rms(h @ p["q"].T, eps) * p["q.norm"]).view(t, heads, m["dim"])
    k = (rms(h @ p["k"].T, eps) * p["k.norm"]).view(t, g, m["dim"])
    v = rms((h @ p["v"].T).view(t, g, m["vdim"]), eps)
    if past is not None:
        k, v = torch.cat([past[0], k]), torch.cat([past[1], v])
    o = chunk_attend(q, k, v, m["scale"], m["mask"]["size"])
    return o.reshape(t, -1) @ p["o"].T, (k, v)


def hgrn_recurrence(q, f, v, state):
    """q, f [T, H, d]; v [T, H, e]; state [H, d, e].  What the gate lets go of is what is written."""
    out, s = [], state
    for t in range(q.shape[0]):
        s = f[t][:, :, None] * s + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        out.append((s * q[t][:, :, None]).sum(1))
    return torch.stack(out), s


def hgrn_mixer(h, p, m, eps, past):
    t, heads, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    if past is None:
        past = torch.zeros(heads, d, e, dtype=F)
    low = p["lower"]
    f = low + (1.0 - low) * sigmoid(h @ p["f"].T + p["f.b"])
    o, past = hgrn_recurrence(silu(h @ p["q"].T).view(t, heads, d), f.view(t, heads, d), (h @ p["v"].T).view(t, heads, e), past)
    return (rms(o, eps) * p["norm"]).reshape(t, heads * e) @ p["o"].T, past


def parallel_mixer(h, p, m, eps, past):
    sub = lambda side: {k[len(side) + 1:]: v for k, v in p.items() if k.startswith(side + ".")}
    past = past or (None, None)
    left, a = attention_mixer(h, sub("left"), m["left"], eps, past[0])
    right, b = hgrn_mixer(h, sub("right"), m["right"], eps, past[1])
    return m["left_scale"] * left + m["right_scale"] * right, (a, b)


def short_conv(x, taps, bias, before):
    """Causal convolution over time per channel, then silu.  x [T, C], taps [C, n] (last column: the current token),
    before [n - 1, C]: the inputs ahead of x.  Returns (output, the last n - 1 inputs)."""
    n = taps.shape[1]
    full = torch.cat([before, x])
    y = sum(full[j:j + x.shape[0]] * taps[:, j] for j in range(n)) + bias
    return silu(y), full[full.shape[0] - (n - 1):]


def mamba_recurrence(x, b, c, dt, a_log, skip, state):
    """x [T, H, e]; b, c [T, H, N]; dt [T, H]; state [H, N, e]."""
    out, s = [], state
    for t in range(x.shape[0]):
        keep = torch.exp(-torch.exp(a_log) * dt[t])
        s = keep[:, None, None] * s + dt[t][:, None, None] * b[t][:, :, None] * x[t][:, None, :]
        out.append((s * c[t][:, :, None]).sum(1) + skip[:, None] * x[t])
    return torch.stack(out), s


def mamba_mixer(h, p, m, eps, past):
    """past: None or (the convolution's last inputs, S)."""
    t, heads, e, groups, n = h.shape[0], m["heads"], m["vdim"], m["groups"], m["state"]
    inner = heads * e
    z, xbc, dt = (h @ p["in"].T).split([inner, inner + 2 * groups * n, heads], 1)
    if past is None:
        past = (torch.zeros(m["conv"] - 1, xbc.shape[1], dtype=F), torch.zeros(heads, n, e, dtype=F))
    xbc, keep = short_conv(xbc, p["conv"], p["conv.b"], past[0])
    x, b, c = xbc.split([inner, groups * n, groups * n], 1)
    spread = lambda y: torch.stack([y.view(t, groups, n)[:, i // (heads // groups)] for i in range(heads)], 1)
    y, s = mamba_recurrence(x.view(t, heads, e), spread(b), spread(c), softplus(dt + p["dt_bias"]), p["A_log"], p["D"], past[1])
    y = y.reshape(t, inner) * silu(z)
    y = rms(y.view(t, m["norm_groups"], -1), eps).reshape(t, inner) * p["norm"]
    return y @ p["o"].T, (keep, s)


MIXERS = {"mlstm": mlstm_mixer, "parallel": parallel_mixer, "mamba2": mamba_mixer}


# ----------------------------------------------------------------------------------------------- feed-forward
def gated(h, p, prefix):
    return (silu(h @ p[prefix + ".gate"].T) * (h @ p[prefix + ".up"].T)) @ p[prefix + ".down"].T


def choose(z, correction, top, scale):
    """Router logits [T, E] -> (chosen ids [T, top], weights [T, top])."""
    s = torch.softmax(z, -1)
    idx = torch.sort(s + correction, dim=-1, descending=True, stable=True).indices[:, :top]
    return idx, torch.gather(s, 1, idx) * scale


def experts_ff(h, p, m):
    r = m["router"]
    idx, w = choose(h @ p["router"].T, p["correction"], r["top"], r["scale"])
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, x in zip(idx[t].tolist(), w[t]):
            y[t] += x * (gated(h[t:t + 1], p, f"e{e}")[0] if e < r["experts"] else h[t])
    return y + gated(h, p, "shared")


# ----------------------------------------------------------------------------------------------- the whole model
class PlainZazilix:
    """One sequence: ``step(tokens)`` returns the logits of every new token and keeps what every layer remembers."""

    def __init__(self, cfg: dict, tensors: dict):
        self.cfg = cfg
        self.w = {k: v.to(F) for k, v in tensors.items()}
        self.eps = cfg["norm"]["eps"]
        self.reset()

    def reset(self):
        self.memory, self.length = {}, 0
        self.residuals = []       # the sum of the streams after every layer of the last step

    def _sub(self, prefix):
        return {k[len(prefix):]: v for k, v in self.w.items() if k.startswith(prefix)}

    def _norm(self, x, name):
        return rms(x, self.eps) * self.w[name]

    def step(self, tokens):
        t, w = len(tokens), self.w
        x = w["embed"][torch.as_tensor(tokens, dtype=torch.int64)] * self.cfg["embedding"]["scale"]
        x = x + w["pos"][self.length:self.length + t]
        self.length += t
        x = torch.stack([x] * self.cfg["streams"])
        self.residuals = []
        for i, layer in enumerate(self.cfg["layers"]):
            l = f"l{i}."
            h = self._norm(stream_in(x, w[l + "hc1.in"]), l + "norm1")
            y, self.memory[i] = MIXERS[layer["type"]](h, self._sub(l + "mix."), layer["mixer"], self.eps, self.memory.get(i))
            x = stream_out(x, w[l + "hc1.mix"], w[l + "hc1.out"], y)
            if layer.get("mlp") is not None:
                h = self._norm(stream_in(x, w[l + "hc2.in"]), l + "norm2")
                x = stream_out(x, w[l + "hc2.mix"], w[l + "hc2.out"], experts_ff(h, self._sub(l + "mlp."), layer["mlp"]))
            self.residuals.append(x.sum(0))
        return self._norm(x.sum(0), "final.norm") @ w["head"].T


# ----------------------------------------------------------------------------------------------- small random models
def mlstm_layer(heads=3, dim=24, vdim=16, cap=9.0, ff=None):
    return {"type": "mlstm", "mlp": ff, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def parallel_layer(heads=6, kv_heads=3, dim=16, vdim=24, size=50, scale=0.3, rheads=2, rdim=24, rvdim=32, left=0.8, right=1.3,
                   ff=None):
    return {"type": "parallel", "mlp": ff,
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                               "mask": {"size": size}},
                      "right": {"heads": rheads, "dim": rdim, "vdim": rvdim}, "left_scale": left, "right_scale": right}}


def mamba_layer(heads=4, vdim=24, groups=2, state=16, conv=3, norm_groups=4, ff=None):
    return {"type": "mamba2", "mlp": ff, "mixer": {"heads": heads, "vdim": vdim, "groups": groups, "state": state, "conv": conv,
                                                   "norm_groups": norm_groups}}


def moe(ff=40, experts=6, top=3, identity=2, scale=1.7, shared=56):
    return {"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": shared},
            "router": {"experts": experts, "top": top, "identity": identity, "scale": scale}}


def config(layers, width=96, vocab=136, streams=3, scale=1.5, eps=2e-5, positions=1024):
    return {"architecture": "Zazilix", "layers": layers, "width": width, "vocab": vocab, "streams": streams,
            "embedding": {"scale": scale}, "norm": {"eps": eps}, "max_positions": positions}


def tensors(cfg, seed=0, clear=False):
    """Random tensors of the configuration in the checkpoint's names (bfloat16).  clear: the routers' corrections alone decide which
    experts are chosen, so that rounding never does."""
    g = torch.Generator().manual_seed(seed)
    width, n, out = cfg["width"], cfg["streams"], {}

    def lin(name, rows, cols, gain=1.0):
        out[name] = torch.randn(rows, cols, generator=g) * gain / math.sqrt(cols)

    def vec(name, size, std=0.3, mean=0.0):
        out[name] = torch.randn(size, generator=g) * std + mean

    def scalar(name):
        out[name] = torch.rand((), generator=g) + 0.5

    def connections(name):
        vec(name + ".in", n, 0.3, 1.0 / n)
        vec(name + ".out", n, 0.3, 1.0)
        out[name + ".mix"] = torch.eye(n) * 0.8 + torch.randn(n, n, generator=g) * 0.12

    out["embed"] = torch.randn(cfg["vocab"], width, generator=g)
    out["pos"] = torch.randn(cfg["max_positions"], width, generator=g) * 0.4
    lin("head", cfg["vocab"], width)
    scalar("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        p, m, kind = f"l{i}.", layer["mixer"], layer["type"]
        q = p + "mix."
        scalar(p + "norm1")
        connections(p + "hc1")
        if kind == "mlstm":
            h = m["heads"]
            lin(q + "q", h * m["dim"], width, 2.0)
            lin(q + "k", h * m["dim"], width, 0.6)
            out[q + "k"] += 0.4 * out[q + "q"]       # a token answers its own query: a head's output is no small difference
            lin(q + "v", h * m["vdim"], width)
            lin(q + "g", h * m["vdim"], width, 2.0)
            lin(q + "o", width, h * m["vdim"])
            vec(q + "norm", h * m["vdim"], 0.2, 1.0)
            lin(q + "i", h, width, 2.0)
            vec(q + "i.b", h, 1.0, -1.0)
            lin(q + "f", h, width, 2.0)
            vec(q + "f.b", h, 1.0, 4.0)
        elif kind == "parallel":
            a, r = m["left"], m["right"]
            lin(q + "left.q", a["heads"] * a["dim"], width)
            lin(q + "left.k", a["kv_heads"] * a["dim"], width)
            lin(q + "left.v", a["kv_heads"] * a["vdim"], width)
            vec(q + "left.q.norm", a["heads"] * a["dim"], 0.3, 1.5)
            vec(q + "left.k.norm", a["kv_heads"] * a["dim"], 0.3, 1.5)
            lin(q + "left.o", width, a["heads"] * a["vdim"])
            lin(q + "right.q", r["heads"] * r["dim"], width, 2.0)
            lin(q + "right.f", r["heads"] * r["dim"], width, 2.0)
            vec(q + "right.f.b", r["heads"] * r["dim"], 1.0, 2.0)
            out[q + "right.lower"] = torch.rand(r["heads"] * r["dim"], generator=g) * 0.9
            lin(q + "right.v", r["heads"] * r["vdim"], width)
            vec(q + "right.norm", r["vdim"], 0.2, 1.0)
            lin(q + "right.o", width, r["heads"] * r["vdim"])
        else:
            h = m["heads"]
            inner, c = h * m["vdim"], h * m["vdim"] + 2 * m["groups"] * m["state"]
            lin(q + "in", inner + c + h, width, 1.5)
            out[q + "conv"] = torch.randn(c, m["conv"], generator=g) * (0.7 / math.sqrt(m["conv"])) + 0.3
            vec(q + "conv.b", c, 0.3)
            vec(q + "dt_bias", h, 1.0, -2.0)
            out[q + "A_log"] = torch.rand(h, generator=g) * 3.0 - 2.0
            vec(q + "D", h, 0.5, 1.0)
            vec(q + "norm", inner, 0.2, 1.0)
            lin(q + "o", width, inner)
        ff = layer.get("mlp")
        if ff is not None:
            scalar(p + "norm2")
            connections(p + "hc2")
            r, q = ff["router"], p + "mlp."
            lin(q + "router", r["experts"] + r["identity"], width, 2.0)
            vec(q + "correction", r["experts"] + r["identity"], 0.1)
            if clear:
                out[q + "correction"] = torch.randperm(r["experts"] + r["identity"], generator=g) * 1.5
            for name, size in [(f"e{e}", ff["expert"]["ff"]) for e in range(r["experts"])] + [("shared", ff["shared"]["ff"])]:
                lin(f"{q}{name}.gate", size, width, 1.5)
                lin(f"{q}{name}.up", size, width)
                lin(f"{q}{name}.down", width, size)
    return {k: v.to(torch.bfloat16) for k, v in out.items()}


def write_model(cfg, tens, folder):
    from safetensors.torch import save_file

    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in tens.items()}, os.path.join(folder, "model.safetensors"))
    return str(folder)
