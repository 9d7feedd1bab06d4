"""Plain, slow statement of the Buvalix design on the CPU, in float64, one function per mechanism and one sequence at a
time.  It is written from the design's equations and shares no code with the package; the tests compare the package with
it.  Also makes small random models (configuration dict + tensors) in the checkpoint's own names and layout."""
import json
import math
import os

import torch

F = torch.float64


# ----------------------------------------------------------------------------------------------- mechanisms
def layer_norm(x, w, b, eps):
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w + b


def gelu_tanh(x):
    return 0.5 * x * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def rotate(x, positions, dims, base):
    """x [T, heads, dim]: neighbouring pairs of the first ``dims`` dimensions turn by position * base^(-2i/dims)."""
    out = x.clone()
    for i in range(dims // 2):
        a = positions.to(F) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i], out[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def query_temperature(position, coef, every):
    return 1.0 + coef * math.log((position + 1) // every + 1)


def distance_bucket(n, rows, limit):
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + int(math.floor(math.log(n / half) / math.log(limit / half) * (rows - half))))


def softcap(s, cap):
    return cap * torch.tanh(s / cap)


def attend(q, k, v, group, scale, cap, sink, bias):
    """q [T, H, dim] at the last T places of k [n, G, dim], v [n, G, vdim]; query head h reads key head h // group.  sink
    [H] or None; bias(distances) -> [.., H] or None."""
    t, heads = q.shape[:2]
    n = k.shape[0]
    away = (n - t + torch.arange(t))[:, None] - torch.arange(n)[None, :]          # [T, n], negative: not seen
    out = []
    for h in range(heads):
        s = softcap(q[:, h] @ k[:, h // group].T * scale, cap)
        if bias is not None:
            s = s + bias(away.clamp_min(0))[..., h]
        s = torch.where(away >= 0, s, torch.full_like(s, -math.inf))
        top = s.max(-1, keepdim=True).values
        if sink is not None:
            top = torch.maximum(top, sink[h])
        e = torch.exp(s - top)
        total = e.sum(-1, keepdim=True) + (0.0 if sink is None else torch.exp(sink[h] - top))
        out.append((e / total) @ v[:, h // group])
    return torch.stack(out, 1)


def rotary_attention_mixer(h, p, m, past):
    """Biased projections, rotation, capped scores, softmax with a sink.  past: None or (keys, values)."""
    t, heads, g = h.shape[0], m["heads"], m["kv_heads"]
    n0 = 0 if past is None else past[0].shape[0]
    pos = torch.arange(n0, n0 + t)
    q, k, v = (h @ p[n].T + p[n + ".b"] for n in ("q", "k", "v"))
    q = rotate(q.view(t, heads, m["dim"]), pos, m["rot"]["dims"], m["rot"]["base"])
    k = rotate(k.view(t, g, m["dim"]), pos, m["rot"]["dims"], m["rot"]["base"])
    v = v.view(t, g, m["vdim"])
    if past is not None:
        k, v = torch.cat([past[0], k]), torch.cat([past[1], v])
    o = attend(q, k, v, heads // g, m["scale"], m["softcap"], p["sink"], None)
    return o.reshape(t, -1) @ p["o"].T, (k, v)


def bucket_attention_mixer(h, p, m, past):
    """No rotation: query temperature by position, capped scores, a learned bias per distance bucket."""
    t, heads, g = h.shape[0], m["heads"], m["kv_heads"]
    n0 = 0 if past is None else past[0].shape[0]
    q, k, v = (h @ p[n].T for n in ("q", "k", "v"))
    temp = torch.tensor([query_temperature(n0 + i, m["q_temp"]["coef"], m["q_temp"]["every"]) for i in range(t)], dtype=F)
    q = q.view(t, heads, m["dim"]) * temp[:, None, None]
    k, v = k.view(t, g, m["dim"]), v.view(t, g, m["vdim"])
    if past is not None:
        k, v = torch.cat([past[0], k]), torch.cat([past[1], v])
    rows = p["rel"].shape[0]
    table = torch.stack([p["rel"][distance_bucket(n, rows, m["bias_max"])] for n in range(k.shape[0])])
    o = attend(q, k, v, heads // g, m["scale"], m["softcap"], None, lambda n: table[n])
    return o.reshape(t, -1) @ p["o"].T, (k, v)


def short_conv(x, taps, before):
    """Causal convolution over time per channel, then silu.  x [T, C], taps [C, n] (last column: the current token),
    before [n - 1, C]: the inputs ahead of x.  Returns (output, the last n - 1 inputs)."""
    n = taps.shape[1]
    full = torch.cat([before, x])
    y = sum(full[j:j + x.shape[0]] * taps[:, j] for j in range(n))
    return y * sigmoid(y), full[full.shape[0] - (n - 1):]


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_recurrence(q, k, v, g, beta, state):
    """q, k, g [T, H, d]; v [T, H, e]; beta [T, H]; state [H, d, e].  Token by token."""
    out, s = [], state.clone()
    for t in range(q.shape[0]):
        s = g[t][:, :, None] * s
        u = beta[t][:, None] * (v[t] - (s * k[t][:, :, None]).sum(1))
        s = s + k[t][:, :, None] * u[:, None, :]
        out.append((s * q[t][:, :, None]).sum(1))
    return torch.stack(out), s


def delta_inputs(h, p, m, before):
    """(q, k, v, g, beta, the convolutions' last inputs) of the recurrence; before: name -> inputs ahead of h."""
    t, heads, kvh, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    conv, keep = {}, {}
    for n in "qkv":
        conv[n], keep[n] = short_conv(h @ p[n].T, p[n + ".conv"], before[n])
    spread = lambda x: x.view(t, kvh, d).repeat_interleave(heads // kvh, 1)
    q, k = unit(spread(conv["q"])) / math.sqrt(d), unit(spread(conv["k"]))
    rate = h @ p["a1"].T @ p["a2"].T + p["dt_bias"]
    soft = torch.log1p(torch.exp(-rate.abs())) + rate.clamp_min(0)
    g = torch.exp(-torch.exp(p["A_log"])[:, None] * soft.view(t, heads, d))
    return q, k, conv["v"].view(t, heads, e), g, sigmoid(h @ p["b"].T), keep


def delta_mixer(h, p, m, eps, past):
    """past: None or (convolution inputs, S [H, d, e])."""
    t, heads, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    if past is None:
        past = ({n: torch.zeros(m["conv"] - 1, p[n].shape[0], dtype=F) for n in "qkv"}, torch.zeros(heads, d, e, dtype=F))
    q, k, v, g, beta, keep = delta_inputs(h, p, m, past[0])
    o, s = delta_recurrence(q, k, v, g, beta, past[1])
    o = o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps) * p["norm"]
    y = o.reshape(t, heads * e) * sigmoid(h @ p["g1"].T @ p["g2"].T)
    return y @ p["o"].T, (keep, s)


def gated_ff(h, p):
    return (gelu_tanh(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


# ----------------------------------------------------------------------------------------------- the whole model
class PlainBuvalix:
    """One sequence: ``step(tokens)`` returns the logits of every new token and keeps the caches of every layer run."""

    def __init__(self, cfg: dict, tensors: dict):
        self.cfg = cfg
        self.w = {k: v.to(F) for k, v in tensors.items()}
        self.eps = cfg["norm"]["eps"]
        self.reset()

    def reset(self):
        self.memory = {}
        self.residuals = []       # the residual stream after every layer run of the last step

    def _sub(self, prefix):
        return {k[len(prefix):]: v for k, v in self.w.items() if k.startswith(prefix)}

    def _norm(self, x, name):
        return layer_norm(x, self.w[name], self.w[name + ".b"], self.eps)

    def order(self):
        """(layer, pass or None) in the order they run."""
        n, loop = len(self.cfg["layers"]), self.cfg.get("loop")
        if not loop:
            return [(i, None) for i in range(n)]
        a, b = loop["start"], loop["stop"]
        return ([(i, None) for i in range(a)] + [(i, t) for t in range(loop["times"]) for i in range(a, b)]
                + [(i, None) for i in range(b, n)])

    def step(self, tokens):
        x0 = x = self.w["embed"][torch.as_tensor(tokens, dtype=torch.int64)]
        self.residuals = []
        for run, (i, t) in enumerate(self.order()):
            if t and i == self.cfg["loop"]["start"]:
                x = x + x0
            layer, p = self.cfg["layers"][i], self._sub(f"l{i}.mix.")
            h, m, past = self._norm(x, f"l{i}.norm1"), layer["mixer"], self.memory.get(run)
            if layer["type"] == "attention":
                y, self.memory[run] = rotary_attention_mixer(h, p, m, past)
            elif layer["type"] == "attention_2":
                y, self.memory[run] = bucket_attention_mixer(h, p, m, past)
            else:
                y, self.memory[run] = delta_mixer(h, p, m, self.eps, past)
            x = x + self._norm(y, f"l{i}.norm1b")
            if layer.get("mlp") is not None:
                y = gated_ff(self._norm(x, f"l{i}.norm2"), self._sub(f"l{i}.mlp."))
                x = x + self._norm(y, f"l{i}.norm2b")
            self.residuals.append(x)
        return self._norm(x, "final.norm") @ self.w["head"].T


# ----------------------------------------------------------------------------------------------- small random models
def rotary_layer(heads=4, kv_heads=2, dim=24, vdim=40, rot=16, base=5000.0, scale=0.25, cap=12.0, ff=72):
    return {"type": "attention", "mlp": dense(ff),
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": cap,
                      "rot": {"dims": rot, "base": base}}}


def bucket_layer(heads=6, kv_heads=3, dim=16, vdim=24, limit=100, coef=0.4, every=24, scale=0.3, cap=9.0, ff=40):
    return {"type": "attention_2", "mlp": dense(ff),
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": cap,
                      "bias_max": limit, "q_temp": {"coef": coef, "every": every}}}


def delta_layer(heads=4, kv_heads=2, dim=16, vdim=24, conv=3, ff=None):
    return {"type": "channel_delta", "mlp": dense(ff),
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def dense(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def config(layers, width=96, vocab=136, loop=None, eps=2e-5):
    return {"architecture": "Buvalix", "layers": layers, "width": width, "vocab": vocab, "loop": loop, "norm": {"eps": eps}}


def tensors(cfg, seed=0, rank=12, buckets=20):
    """Random tensors of the configuration in the checkpoint's names (bfloat16).  rank: inner size of the decay's two
    projections, the gate's is four more; buckets: rows of the distance tables (two less for every further layer)."""
    g = torch.Generator().manual_seed(seed)
    width, out = cfg["width"], {}

    def lin(name, n, k, gain=1.0):
        out[name] = torch.randn(n, k, generator=g) * gain / math.sqrt(k)

    def vec(name, n, std=0.3, mean=0.0):
        out[name] = torch.randn(n, generator=g) * std + mean

    def norm(name):
        vec(name, width, 0.3, 1.0)
        vec(name + ".b", width, 0.2)

    out["embed"] = torch.randn(cfg["vocab"], width, generator=g)
    lin("head", cfg["vocab"], width)
    norm("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        q, heads, kvh = p + "mix.", m["heads"], m["kv_heads"]
        norm(p + "norm1")
        norm(p + "norm1b")
        lin(q + "q", (kvh if layer["type"] == "channel_delta" else heads) * m["dim"], width, 2.0)
        lin(q + "k", kvh * m["dim"], width, 2.0)
        lin(q + "v", (heads if layer["type"] == "channel_delta" else kvh) * m["vdim"], width)
        lin(q + "o", width, heads * m["vdim"])
        if layer["type"] == "attention":
            for n in "qkv":
                vec(q + n + ".b", out[q + n].shape[0], 0.5)
            vec(q + "sink", heads, 1.0, 2.0)
        elif layer["type"] == "attention_2":
            out[q + "rel"] = torch.randn(max(buckets - 2 * i, 4), heads, generator=g)
        else:
            for n in "qkv":
                c = out[q + n].shape[0]
                out[q + n + ".conv"] = torch.randn(c, m["conv"], generator=g) * (0.7 / math.sqrt(m["conv"])) + 0.3
            lin(q + "b", heads, width, 1.5)
            out[q + "A_log"] = torch.rand(heads, generator=g) * 3.0 - 2.5
            lin(q + "a1", rank, width)
            lin(q + "a2", heads * m["dim"], rank)
            vec(q + "dt_bias", heads * m["dim"], 1.0, -2.5)
            lin(q + "g1", rank + 4, width)
            lin(q + "g2", heads * m["vdim"], rank + 4, 2.0)
            vec(q + "norm", m["vdim"], 0.2, 1.0)
        ff = layer.get("mlp")
        if ff is not None:
            norm(p + "norm2")
            norm(p + "norm2b")
            lin(p + "mlp.gate", ff["ff"], width, 1.5)
            lin(p + "mlp.up", ff["ff"], width)
            lin(p + "mlp.down", width, ff["ff"])
    return {k: v.to(torch.bfloat16) for k, v in out.items()}


def write_model(cfg, tens, folder):
    from safetensors.torch import save_file

    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in tens.items()}, os.path.join(folder, "model.safetensors"))
    return str(folder)


def rel_err(got, want):
    """Root mean square difference over the root mean square of what is wanted, worst row."""
    got, want = got.to(F).cpu(), want.to(F)
    d = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt().clamp_min(1e-12)
    return float(d.max()) if d.numel() else 0.0
