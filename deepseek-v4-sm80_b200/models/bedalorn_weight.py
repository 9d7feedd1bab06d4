"""Checkpoint loading for the Bedalorn design: raw tensor names -> the tensors its layers run on.

Matrices stay in the checkpoint's bf16 (in 32-bit serving too: the kernels widen them in registers).  Vectors that enter
32-bit computations become fp32, gains stored around zero become 1 + w.  Merged or re-laid for the kernels:

  * ``[q; dkv] -> qc`` (one projection), ``uk`` also transposed per head (``uk_t`` [H*R, dim], absorbed into the query);
  * ``r, k, v, g -> rkvg`` side by side, the five mixes as one [5, D] table in the order r, k, v, g, w;
  * experts -> ``w13`` [E, 2, F, D] (gate, up) and ``w2`` [E, D, F];
  * ``loop.in`` -> its x half and its embedding half (the second product is the same for every pass).
"""
from __future__ import annotations

from typing import Callable, Dict

import torch

from .bedalorn_config import BedalornConfig, DenseSpec, LatentAttentionSpec
from .weight import tensor_reader

MIXES = ("r", "k", "v", "g", "w")


def raw_shapes(cfg: BedalornConfig, decay_rank: int = 64) -> Dict[str, tuple]:
    """Names and shapes of the checkpoint's tensors (``decay_rank``: the inner size of the decay's two projections, the
    one size that only the tensors give)."""
    d = cfg.hidden_size
    out = {"embed": (cfg.vocab_size, d), "final.norm": (d,)}
    if cfg.loop:
        out["loop.in"], out["loop.step"] = (d, 2 * d), (cfg.loop.times, d)
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        out[p + "norm1"] = (d,)
        if isinstance(m, LatentAttentionSpec):
            h, r = m.heads, m.kv_rank
            out.update({p + "mix.q": (h * m.dim, d), p + "mix.dkv": (r, d), p + "mix.dkv.norm": (r,),
                        p + "mix.uk": (h * m.dim, r), p + "mix.uv": (h * m.vdim, r), p + "mix.o": (d, h * m.vdim)})
        else:
            hd = m.heads * m.dim
            out.update({p + "mix.mu." + n: (d,) for n in MIXES})
            out.update({p + "mix." + n: (hd, d) for n in "rkvg"})
            out.update({p + "mix.w1": (decay_rank, d), p + "mix.w2": (hd, decay_rank), p + "mix.w0": (hd,),
                        p + "mix.u": (m.heads, m.dim), p + "mix.norm": (hd,), p + "mix.o": (d, hd)})
        f = l.ff
        if f is None:
            continue
        out[p + "norm2"] = (d,)
        if isinstance(f, DenseSpec):
            out[p + "mlp.up"], out[p + "mlp.down"] = (f.ff, d), (d, f.ff)
        else:
            out[p + "mlp.router"], out[p + "mlp.router.b"] = (f.experts, d), (f.experts,)
            for e in range(f.experts):
                out[f"{p}mlp.e{e}.gate"] = out[f"{p}mlp.e{e}.up"] = (f.ff, d)
                out[f"{p}mlp.e{e}.down"] = (d, f.ff)
    return out


def build_weights(cfg: BedalornConfig, get: Callable[[str], torch.Tensor], device) -> Dict[str, torch.Tensor]:
    """``get(name)`` returns a raw tensor; shapes are checked against the configuration."""
    d = cfg.hidden_size
    want = raw_shapes(cfg)

    def raw(name):
        t = get(name)
        shape = want[name]
        if name.endswith(("mix.w1", "mix.w2")):    # the decay's inner size comes from the tensor
            ok = t.dim() == 2 and (t.shape[1] == d if name.endswith("w1") else t.shape[0] == shape[0])
        else:
            ok = tuple(t.shape) == shape
        if not ok:
            raise ValueError(f"{name}: shape {tuple(t.shape)} does not fit the configuration ({shape})")
        return t

    mat = lambda name: raw(name).to(torch.bfloat16).to(device).contiguous()
    vec = lambda name: raw(name).to(device).float().reshape(-1).contiguous()
    gain = lambda name: vec(name) + 1.0            # stored around zero
    w: Dict[str, torch.Tensor] = {"embed.weight": mat("embed"), "final.gain": gain("final.norm")}
    if cfg.loop:
        inn = mat("loop.in")
        w["loop.in_x"], w["loop.in_x0"] = inn[:, :d].contiguous(), inn[:, d:].contiguous()
        w["loop.step"] = raw("loop.step").to(device).float().contiguous()
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        q = p + "mix."
        w[p + "norm1.gain"] = gain(p + "norm1")
        if isinstance(m, LatentAttentionSpec):
            w[q + "qc"] = torch.cat([mat(q + "q"), mat(q + "dkv")], 0)
            w[q + "latent.gain"] = vec(q + "dkv.norm")
            uk = w[q + "uk"] = mat(q + "uk")
            w[q + "uk_t"] = uk.view(m.heads, m.dim, m.kv_rank).transpose(1, 2).reshape(-1, m.dim).contiguous()
            w[q + "uv"] = mat(q + "uv")
        else:
            w[q + "mu"] = torch.stack([vec(q + "mu." + n) for n in MIXES])
            w[q + "rkvg"] = torch.cat([mat(q + n) for n in "rkvg"], 0)
            w[q + "w1"], w[q + "w2"] = mat(q + "w1"), mat(q + "w2")
            w[q + "w0"], w[q + "u"], w[q + "out.gain"] = vec(q + "w0"), vec(q + "u"), vec(q + "norm")
        w[q + "o"] = mat(q + "o")
        f = l.ff
        if f is None:
            continue
        w[p + "norm2.gain"] = gain(p + "norm2")
        q = p + "mlp."
        if isinstance(f, DenseSpec):
            w[q + "up"], w[q + "down"] = mat(q + "up"), mat(q + "down")
        else:
            w[q + "router"], w[q + "router.b"] = mat(q + "router"), vec(q + "router.b")
            w13 = torch.empty(f.experts, 2, f.ff, d, dtype=torch.bfloat16, device=device)
            w2 = torch.empty(f.experts, d, f.ff, dtype=torch.bfloat16, device=device)
            for e in range(f.experts):
                w13[e, 0], w13[e, 1] = mat(f"{q}e{e}.gate"), mat(f"{q}e{e}.up")
                w2[e] = mat(f"{q}e{e}.down")
            w[q + "w13"], w[q + "w2"] = w13, w2
    return w


def load_checkpoint(folder: str, cfg: BedalornConfig, device) -> Dict[str, torch.Tensor]:
    """Streams a safetensors checkpoint into runtime tensors on ``device``."""
    return build_weights(cfg, tensor_reader(folder), device)


def random_weights(cfg: BedalornConfig, device, seed: int = 0, decay_rank: int = 64) -> Dict[str, torch.Tensor]:
    """Random-init weights: matrices of standard deviation 1 / sqrt(fan-in), gains near one, decays between about 0.6
    and 0.999 per token."""
    shapes = raw_shapes(cfg, decay_rank)
    g = torch.Generator(device=device)
    g.manual_seed(seed * 1000003 + 11)

    def draw(name):
        s = shapes[name]
        r = lambda std: torch.randn(*s, generator=g, device=device, dtype=torch.float32) * std
        if name == "embed" or name.endswith(".u"):
            t = r(1.0 if name == "embed" else 0.5)
        elif name.endswith("mix.w0"):
            t = torch.rand(*s, generator=g, device=device) * 6.0 - 7.0
        elif ".mu." in name:
            t = torch.rand(*s, generator=g, device=device)
        elif name.endswith(("mix.norm", "dkv.norm")):
            t = r(0.1) + 1.0
        elif len(s) == 1 or name == "loop.step":
            t = r(0.1)
        else:
            t = r(s[-1] ** -0.5)
        return t.to(torch.bfloat16)

    return build_weights(cfg, draw, device)
