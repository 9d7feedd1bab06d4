"""Plain, slow statement of the Bedalorn design on the CPU, in float64, one function per mechanism and one sequence at
a time.  It is written from the design's equations and shares no code with the package; the tests compare the package
with it.  Also makes small random models (configuration dict + tensors) in the checkpoint's own names and layout."""
import json
import math
import os

import torch

F = torch.float64


# ----------------------------------------------------------------------------------------------- mechanisms
def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_zero_centred(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def silu(x):
    return x / (1.0 + torch.exp(-x))


def token_shift(h, prev):
    """Rows of h moved down by one; the first row is ``prev`` (what came before this portion)."""
    return torch.cat([prev[None], h[:-1]], 0)


def wkv_recurrence(r, k, v, w, u, state):
    """r, k, v, w [T, H, d]; u [H, d]; state [H, d (key), d (value)].  Token by token."""
    out = []
    s = state.clone()
    for t in range(r.shape[0]):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out.append(((s + u[:, :, None] * kv) * r[t][:, :, None]).sum(1))
        s = w[t][:, :, None] * s + kv
    return torch.stack(out) if out else r, s


def wkv_mixer(h, p, heads, eps, state):
    """h [T, D]; p: name -> tensor; state: None or (previous h [D], S [H, d, d]).  Returns (output, new state)."""
    t, width = h.shape
    hd = p["r"].shape[0]
    d = hd // heads
    prev, s = state if state is not None else (torch.zeros(width, dtype=F), torch.zeros(heads, d, d, dtype=F))
    hp = token_shift(h, prev)
    mix = {n: h + (hp - h) * p["mu." + n] for n in "rkvgw"}
    r, k, v = ((mix[n] @ p[n].T).view(t, heads, d) for n in "rkv")
    gate = silu(mix["g"] @ p["g"].T)
    decay = torch.exp(-torch.exp(torch.tanh(mix["w"] @ p["w1"].T) @ p["w2"].T + p["w0"])).view(t, heads, d)
    o, s = wkv_recurrence(r, k, v, decay, p["u"], s)
    y = rms(o, eps).reshape(t, hd) * p["norm"] * gate
    return y @ p["o"].T, (h[-1], s)


def latent_attention_mixer(h, p, heads, dim, vdim, scale, eps, past):
    """past: None or the latents [n, R] of the tokens before this portion.  Returns (output, all latents)."""
    t = h.shape[0]
    q = (h @ p["q"].T).view(t, heads, dim)
    c_new = rms(h @ p["dkv"].T, eps) * p["dkv.norm"]
    c = c_new if past is None else torch.cat([past, c_new], 0)
    n0 = c.shape[0] - t
    k = (c @ p["uk"].T).view(-1, heads, dim)
    v = (c @ p["uv"].T).view(-1, heads, vdim)
    out = torch.empty(t, heads, vdim, dtype=F)
    for i in range(t):
        see = n0 + i + 1
        for a in range(heads):
            score = (k[:see, a] @ q[i, a]) * scale
            e = torch.exp(score - score.max())
            out[i, a] = (e / e.sum()) @ v[:see, a]
    return out.reshape(t, heads * vdim) @ p["o"].T, c


def dense_ff(h, p):
    a = torch.clamp(h @ p["up"].T, min=0.0)
    return (a * a) @ p["down"].T


def moe_ff(h, p, experts, top):
    out = torch.zeros_like(h)
    z = h @ p["router"].T + p["router.b"]
    for t in range(h.shape[0]):
        best = sorted(range(experts), key=lambda e: (-float(z[t, e]), e))[:top]
        w = torch.softmax(z[t, best], 0)
        for e, we in zip(best, w):
            act = silu(p[f"e{e}.gate"] @ h[t]) * (p[f"e{e}.up"] @ h[t])
            out[t] += we * (p[f"e{e}.down"] @ act)
    return out


# ----------------------------------------------------------------------------------------------- the whole model
class PlainBedalorn:
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

    def order(self):
        """(layer, pass or None) in the order they run."""
        n, loop = len(self.cfg["layers"]), self.cfg.get("loop")
        if not loop:
            return [(i, None) for i in range(n)]
        a, b = loop["start"], loop["stop"]
        return ([(i, None) for i in range(a)] + [(i, t) for t in range(loop["times"]) for i in range(a, b)]
                + [(i, None) for i in range(b, n)])

    def step(self, tokens):
        cfg, w, eps = self.cfg, self.w, self.eps
        x = w["embed"][torch.as_tensor(tokens, dtype=torch.int64)]
        x0 = x
        self.residuals = []
        for run, (i, t) in enumerate(self.order()):
            if t is not None and i == cfg["loop"]["start"]:
                x = torch.cat([x, x0], -1) @ w["loop.in"].T + w["loop.step"][t]
            layer = cfg["layers"][i]
            m, p = layer["mixer"], self._sub(f"l{i}.mix.")
            h = norm_zero_centred(x, w[f"l{i}.norm1"], eps)
            if layer["type"] == "wkv":
                y, self.memory[run] = wkv_mixer(h, p, m["heads"], eps, self.memory.get(run))
            else:
                y, self.memory[run] = latent_attention_mixer(h, p, m["heads"], m["dim"], m["vdim"], m["scale"], eps,
                                                             self.memory.get(run))
            x = x + y
            ff = layer.get("mlp")
            if ff is not None:
                h = norm_zero_centred(x, w[f"l{i}.norm2"], eps)
                p = self._sub(f"l{i}.mlp.")
                x = x + (dense_ff(h, p) if ff["kind"] == "dense"
                         else moe_ff(h, p, ff["router"]["experts"], ff["router"]["top"]))
            self.residuals.append(x)
        x = norm_zero_centred(x, w["final.norm"], eps)
        return (x @ w["embed"].T) * cfg["logit_scale"]


# ----------------------------------------------------------------------------------------------- small random models
def attention_layer(heads=3, dim=24, vdim=40, kv_rank=48, scale=0.2, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale}}


def wkv_layer(heads=2, dim=16, mlp=None):
    return {"type": "wkv", "mlp": mlp, "mixer": {"heads": heads, "dim": dim}}


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, top=2, ff=40):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(layers, width=96, vocab=136, loop=None, eps=2e-5, logit_scale=1.5):
    return {"architecture": "Bedalorn", "layers": layers, "width": width, "vocab": vocab, "loop": loop,
            "norm": {"eps": eps}, "logit_scale": logit_scale}


def tensors(cfg, seed=0, rank_w=12):
    """Random tensors of the configuration in the checkpoint's names (bfloat16)."""
    g = torch.Generator().manual_seed(seed)
    width, out = cfg["width"], {}

    def lin(name, n, k, gain=1.0):
        out[name] = torch.randn(n, k, generator=g) * gain / math.sqrt(k)

    def vec(name, n, std=0.3, mean=0.0):
        out[name] = torch.randn(n, generator=g) * std + mean

    out["embed"] = torch.randn(cfg["vocab"], width, generator=g)
    vec("final.norm", width)
    if cfg.get("loop"):
        lin("loop.in", width, 2 * width)
        out["loop.step"] = torch.randn(cfg["loop"]["times"], width, generator=g) * 0.5
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        vec(p + "norm1", width)
        h = m["heads"]
        if layer["type"] == "wkv":
            hd = h * m["dim"]
            for n in "rkvgw":
                out[p + "mix.mu." + n] = torch.rand(width, generator=g)
            for n in "rkvg":
                lin(p + "mix." + n, hd, width)
            lin(p + "mix.w1", rank_w, width)
            lin(p + "mix.w2", hd, rank_w)
            out[p + "mix.w0"] = torch.rand(hd, generator=g) * 4.0 - 5.0
            out[p + "mix.u"] = torch.randn(h, m["dim"], generator=g) * 0.5
            vec(p + "mix.norm", hd, 0.2, 1.0)
            lin(p + "mix.o", width, hd)
        else:
            lin(p + "mix.q", h * m["dim"], width, 2.0)
            lin(p + "mix.dkv", m["kv_rank"], width)
            vec(p + "mix.dkv.norm", m["kv_rank"], 0.2, 1.0)
            lin(p + "mix.uk", h * m["dim"], m["kv_rank"])
            lin(p + "mix.uv", h * m["vdim"], m["kv_rank"])
            lin(p + "mix.o", width, h * m["vdim"])
        ff = layer.get("mlp")
        if ff is None:
            continue
        vec(p + "norm2", width)
        if ff["kind"] == "dense":
            lin(p + "mlp.up", ff["ff"], width)
            lin(p + "mlp.down", width, ff["ff"])
        else:
            e, f = ff["router"]["experts"], ff["expert"]["ff"]
            lin(p + "mlp.router", e, width, 3.0)
            vec(p + "mlp.router.b", e, 0.5)
            for j in range(e):
                lin(f"{p}mlp.e{j}.gate", f, width)
                lin(f"{p}mlp.e{j}.up", f, width)
                lin(f"{p}mlp.e{j}.down", width, f)
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
