"""Plain, slow statement of the Sakevik design on the CPU, in float64, one function per mechanism and one sequence at a time.  It
is written from the design's equations and shares no code with the package; the tests compare the package with it.  Also makes
small random models (configuration dict + tensors) in the checkpoint's own names and layout."""
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


def bigram_rows(tokens, before, spec):
    """Row of the bigram table of every token; before: the token ahead of the first one, None at the start of a sequence."""
    rows = []
    for t in tokens:
        n = spec["buckets"]
        rows.append(n if before is None else (int(before) * spec["mul_prev"] + int(t) * spec["mul_cur"]) % n)
        before = t
    return rows


# ----------------------------------------------------------------------------------------------- rotation
def frequencies(rot, dims):
    """(angle per position of every pair, factor of cos and sin)."""
    f = [rot["base"] ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if not s:
        return torch.tensor(f, dtype=F), 1.0
    edge = lambda turns: dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(rot["base"]))
    lo, hi = max(math.floor(edge(s["fast"])), 0), min(math.ceil(edge(s["slow"])), dims - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / s["factor"] * ramp + x * (1.0 - ramp))
    return torch.tensor(out, dtype=F), 0.1 * math.log(s["factor"]) + 1.0


def turn(x, pos, freq, mul, halves, back=False):
    """x [T, heads, n]: the first 2 * len(freq) dimensions turn by position * freq; partners are half of them apart, or neighbours."""
    m = len(freq)
    a = pos.to(F)[:, None, None] * freq * (-1.0 if back else 1.0)
    c, s = torch.cos(a) * mul, torch.sin(a) * mul
    out = x.clone()
    first, second = (slice(0, m), slice(m, 2 * m)) if halves else (slice(0, 2 * m, 2), slice(1, 2 * m, 2))
    u, v = x[..., first], x[..., second]
    out[..., first], out[..., second] = u * c - v * s, v * c + u * s
    return out


# ----------------------------------------------------------------------------------------------- mixers
def mingru_recurrence(z, u, state):
    """z, u [T, n] (gate and candidate input), state [n]."""
    out = []
    for t in range(z.shape[0]):
        cand = torch.where(u[t] >= 0, u[t] + 0.5, sigmoid(u[t]))
        state = (1.0 - z[t]) * state + z[t] * cand
        out.append(state)
    return torch.stack(out), state


def mingru_mixer(h, p, m, eps, past, pos):
    if past is None:
        past = torch.zeros(m["width"], dtype=F)
    s, past = mingru_recurrence(sigmoid(h @ p["z"].T + p["z.b"]), h @ p["x"].T + p["x.b"], past)
    return (s * silu(h @ p["g"].T)) @ p["o"].T, past


def sigmoid_attend(q, k, v, scale, window, bias):
    """q [T, H, d] at the last T places of k [n, G, d], v [n, G, e].  Weights are sigmoids, one key does not know of the others."""
    t, heads = q.shape[:2]
    n, groups = k.shape[:2]
    out = torch.zeros(t, heads, v.shape[2], dtype=F)
    for h in range(heads):
        g = h // (heads // groups)
        for r in range(t):
            i = n - t + r
            lo = max(0, i - window + 1)
            out[r, h] = sigmoid(k[lo:i + 1, g] @ q[r, h] * scale + bias[h]) @ v[lo:i + 1, g]
    return out


def attention_mixer(h, p, m, eps, past, pos):
    """past: None or (keys, values), both as they are cached: the values turned by their positions."""
    t, heads, g, e = h.shape[0], m["heads"], m["kv_heads"], m["vdim"]
    proj = lambda name, n: (h @ p[name].T + p[name + ".b"]).view(t, n, -1)
    freq, mul = frequencies(m["rot"], m["rot"]["dims"])
    vfreq, _ = frequencies({"base": m["rot"]["base"]}, e)
    q = turn(rms(proj("q", heads), eps) * p["q.norm"], pos, freq, mul, True)
    k = turn(rms(proj("k", g), eps) * p["k.norm"], pos, freq, mul, True)
    v = turn(proj("v", g), pos, vfreq, 1.0, True)
    if past is not None:
        k, v = torch.cat([past[0], k]), torch.cat([past[1], v])
    o = turn(sigmoid_attend(q, k, v, m["scale"], m["mask"]["size"], p["pb"]), pos, vfreq, 1.0, True, back=True)
    o = o * sigmoid(h @ p["g"].T)[:, :, None]
    return o.reshape(t, -1) @ p["o"].T + p["o.b"], (k, v)


def softmax_attend(q, k, v, scale, window):
    """q [T, H, d] at the last T places of k [n, H, d], v [n, H, e]."""
    t, heads = q.shape[:2]
    n = k.shape[0]
    out = torch.zeros(t, heads, v.shape[2], dtype=F)
    for h in range(heads):
        for r in range(t):
            i = n - t + r
            lo = max(0, i - window + 1)
            out[r, h] = torch.softmax(k[lo:i + 1, h] @ q[r, h] * scale, 0) @ v[lo:i + 1, h]
    return out


def latent_mixer(h, p, m, eps, past, pos):
    """past: None or (latents, turned key parts), one row of each per token."""
    t, heads, d, r, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    freq, mul = frequencies(m["rot"], r)
    q = (h @ p["q"].T).view(t, heads, d + r)
    q = torch.cat([q[..., :d], turn(q[..., d:], pos, freq, mul, False)], -1)
    down = h @ p["dkv"].T
    c = rms(down[:, :rank], eps) * p["dkv.norm"]
    kr = turn(down[:, None, rank:], pos, freq, mul, False)[:, 0]
    if past is not None:
        c, kr = torch.cat([past[0], c]), torch.cat([past[1], kr])
    n = c.shape[0]
    k = torch.cat([(c @ p["uk"].T).view(n, heads, d), kr[:, None].expand(n, heads, r)], -1)
    o = softmax_attend(q, k, (c @ p["uv"].T).view(n, heads, -1), m["scale"], m["mask"]["size"])
    return o.reshape(t, -1) @ p["o"].T, (c, kr)


MIXERS = {"mingru": mingru_mixer, "attention": attention_mixer, "latent_attention": latent_mixer}


# ----------------------------------------------------------------------------------------------- feed-forward
def clamped_gate(gate, up, limit):
    g, u = gate.clamp(max=limit), up.clamp(-limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def feed_forward(h, p, m):
    return clamped_gate(h @ p["gate"].T, h @ p["up"].T, m["limit"]) @ p["down"].T


# ----------------------------------------------------------------------------------------------- the whole model
class PlainSakevik:
    """One sequence: ``step(tokens)`` returns the logits of every new token and keeps what every layer remembers."""

    def __init__(self, cfg: dict, tensors: dict):
        self.cfg = cfg
        self.w = {k: v.to(F) for k, v in tensors.items()}
        self.eps = cfg["norm"]["eps"]
        self.reset()

    def reset(self):
        self.memory, self.length, self.last = {}, 0, None
        self.residuals = []       # the stream after every layer of the last step

    def _sub(self, prefix):
        return {k[len(prefix):]: v for k, v in self.w.items() if k.startswith(prefix)}

    def step(self, tokens):
        w, emb = self.w, self.cfg["embedding"]
        x = w["embed"][torch.as_tensor(tokens, dtype=torch.int64)] * emb["scale"]
        x = x + w["bigram"][torch.tensor(bigram_rows(tokens, self.last, emb["bigram"]))]
        pos = torch.arange(self.length, self.length + len(tokens))
        self.length, self.last = self.length + len(tokens), tokens[-1]
        self.residuals = []
        for i, layer in enumerate(self.cfg["layers"]):
            l = f"l{i}."
            y, self.memory[i] = MIXERS[layer["type"]](x, self._sub(l + "mix."), layer["mixer"], self.eps, self.memory.get(i), pos)
            x = x + rms(y, self.eps) * w[l + "norm1"]
            if layer.get("mlp") is not None:
                x = x + rms(feed_forward(x, self._sub(l + "mlp."), layer["mlp"]), self.eps) * w[l + "norm2"]
            self.residuals.append(x)
        return (rms(x, self.eps) * w["final.norm"]) @ w["head"].T * self.cfg["logit_scale"]


# ----------------------------------------------------------------------------------------------- small random models
def dense(ff=72, limit=1.2):
    return {"kind": "dense", "ff": ff, "limit": limit}


def mingru_layer(width=80, ff=None):
    return {"type": "mingru", "mlp": ff, "mixer": {"width": width}}


def attention_layer(heads=6, kv_heads=3, dim=32, vdim=24, size=50, dims=24, base=900.0, scale=0.3, ff=None):
    return {"type": "attention", "mlp": ff,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size},
                      "rot": {"base": base, "dims": dims}, "scale": scale}}


def latent_layer(heads=4, dim=24, rot_dim=16, vdim=40, rank=48, size=70, base=3000.0, scale=0.25, scaling=(4.0, 64, 8.0, 1.0), ff=None):
    factor, original, fast, slow = scaling
    return {"type": "latent_attention", "mlp": ff,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "mask": {"size": size},
                      "rot": {"base": base, "dims": rot_dim,
                              "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}},
                      "scale": scale}}


def config(layers, width=96, vocab=136, scale=1.5, eps=2e-5, logit_scale=0.7, buckets=61, mul_prev=7, mul_cur=13):
    return {"architecture": "Sakevik", "layers": layers, "width": width, "vocab": vocab, "logit_scale": logit_scale,
            "embedding": {"scale": scale, "bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}},
            "norm": {"eps": eps}}


def tensors(cfg, seed=0):
    """Random tensors of the configuration in the checkpoint's names (bfloat16)."""
    g = torch.Generator().manual_seed(seed)
    width, out = cfg["width"], {}

    def lin(name, rows, cols, gain=1.0):
        out[name] = torch.randn(rows, cols, generator=g) * gain / math.sqrt(cols)

    def vec(name, size, std=0.3, mean=0.0):
        out[name] = torch.randn(size, generator=g) * std + mean

    out["embed"] = torch.randn(cfg["vocab"], width, generator=g)
    out["bigram"] = torch.randn(cfg["embedding"]["bigram"]["buckets"] + 1, width, generator=g)
    lin("head", cfg["vocab"], width)
    vec("final.norm", width, 0.2, 1.0)
    for i, layer in enumerate(cfg["layers"]):
        p, m, kind = f"l{i}.", layer["mixer"], layer["type"]
        q = p + "mix."
        vec(p + "norm1", width, 0.2, 1.0)
        if kind == "mingru":
            n = m["width"]
            lin(q + "z", n, width)
            vec(q + "z.b", n, 1.5, -1.5)          # tokens to tens of tokens of memory
            lin(q + "x", n, width, 1.5)
            vec(q + "x.b", n)
            lin(q + "g", n, width)
            lin(q + "o", width, n)
        elif kind == "attention":
            nq, nk, nv = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
            for name, n in (("q", nq), ("k", nk), ("v", nv)):
                lin(q + name, n, width)
                vec(q + name + ".b", n)
            vec(q + "q.norm", m["dim"], 0.3, 1.5)
            vec(q + "k.norm", m["dim"], 0.3, 1.5)
            vec(q + "pb", m["heads"], 1.0, -2.5)
            lin(q + "g", m["heads"], width)
            lin(q + "o", width, m["heads"] * m["vdim"])
            vec(q + "o.b", width, 0.1)
        else:
            h, rank = m["heads"], m["kv_rank"]
            lin(q + "q", h * (m["dim"] + m["rot_dim"]), width, 1.5)
            lin(q + "dkv", rank + m["rot_dim"], width)
            vec(q + "dkv.norm", rank, 0.2, 1.0)
            lin(q + "uk", h * m["dim"], rank)
            lin(q + "uv", h * m["vdim"], rank)
            lin(q + "o", width, h * m["vdim"])
        if layer.get("mlp") is not None:
            ff = layer["mlp"]["ff"]
            vec(p + "norm2", width, 0.2, 1.0)
            lin(p + "mlp.gate", ff, width)
            lin(p + "mlp.up", ff, width)
            lin(p + "mlp.down", width, ff)
    return {k: v.to(torch.bfloat16) for k, v in out.items()}


def write_model(cfg, tens, folder):
    from safetensors.torch import save_file

    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in tens.items()}, os.path.join(folder, "model.safetensors"))
    return str(folder)
