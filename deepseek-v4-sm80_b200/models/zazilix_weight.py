"""Checkpoint loading for the Zazilix design: raw tensor names -> the tensors its layers run on.

Matrices stay in the checkpoint's bf16 (in 32-bit serving too: the kernels widen them in registers); vectors become fp32.
Merged or re-laid for the kernels (every part of a merged projection is padded to a multiple of eight rows, so that the column
slices of its result start on 16 bytes):

  * streams: ``hc.in`` and the norm's gain -> ``pre`` [S + 1], ``hc.out`` and ``hc.mix`` -> ``post`` [S + S * S]; the sum of the
    streams ahead of the head is a ``pre`` of ones;
  * mlstm: ``q, k, v, g -> in``, the two gates ``i, f -> gates`` [2 H, D], which are projected to 32-bit floats;
  * parallel: ``left.q | left.k | left.v``, ``right.q`` and ``right.v`` -> ``in``; the norms' weights ``left.qk.norm``; slopes
    and sinks (logit 0) per head;
  * mamba2: the step sizes' rows of ``in`` -> ``dt`` (projected to 32-bit floats); taps as one [taps, channels] table;
  * experts -> ``w13`` [E, 2, F, D] (gate, up) and ``w2`` [E, D, F]; the shared expert's ``gate, up -> gu`` in alternating blocks
    of 16 rows, its size padded to a multiple of 16 with zeros.
"""
from __future__ import annotations

from typing import Callable, Dict

import torch
from torch.nn.functional import pad

from .buvalix_weight import GATE_BLOCK, interleave_gate
from .weight import tensor_reader
from .zazilix_config import MambaSpec, MLSTMSpec, ParallelSpec, ZazilixConfig


def raw_shapes(cfg: ZazilixConfig) -> Dict[str, tuple]:
    """Names and shapes of the checkpoint's tensors."""
    d, n = cfg.hidden_size, cfg.streams
    out: Dict[str, tuple] = {"embed": (cfg.vocab_size, d), "pos": (cfg.position_rows, d), "final.norm": (),
                             "head": (cfg.vocab_size, d)}

    def connections(p, q):
        out.update({f"{p}norm{q}": (), f"{p}hc{q}.in": (n,), f"{p}hc{q}.out": (n,), f"{p}hc{q}.mix": (n, n)})

    def gated(p, ff):
        out.update({p + ".gate": (ff, d), p + ".up": (ff, d), p + ".down": (d, ff)})

    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        q = p + "mix."
        connections(p, 1)
        if isinstance(m, MLSTMSpec):
            hd, he = m.heads * m.dim, m.heads * m.vdim
            out.update({q + "q": (hd, d), q + "k": (hd, d), q + "v": (he, d), q + "g": (he, d), q + "o": (d, he),
                        q + "norm": (he,), q + "i": (m.heads, d), q + "i.b": (m.heads,), q + "f": (m.heads, d),
                        q + "f.b": (m.heads,)})
        elif isinstance(m, ParallelSpec):
            l_, r = m.left, m.right
            nq, nk, rd = l_.heads * l_.dim, l_.kv_heads * l_.dim, r.heads * r.dim
            out.update({q + "left.q": (nq, d), q + "left.k": (nk, d), q + "left.v": (l_.kv_heads * l_.vdim, d),
                        q + "left.q.norm": (nq,), q + "left.k.norm": (nk,), q + "left.o": (d, l_.heads * l_.vdim),
                        q + "right.q": (rd, d), q + "right.f": (rd, d), q + "right.f.b": (rd,), q + "right.lower": (rd,),
                        q + "right.v": (r.heads * r.vdim, d), q + "right.norm": (r.vdim,),
                        q + "right.o": (d, r.heads * r.vdim)})
        else:
            inner = m.heads * m.vdim
            c = inner + 2 * m.groups * m.state
            out.update({q + "in": (inner + c + m.heads, d), q + "conv": (c, m.conv), q + "conv.b": (c,),
                        q + "dt_bias": (m.heads,), q + "A_log": (m.heads,), q + "D": (m.heads,), q + "norm": (inner,),
                        q + "o": (d, inner)})
        if l.ff is not None:
            f, q = l.ff, p + "mlp."
            connections(p, 2)
            out[q + "router"], out[q + "correction"] = (f.experts + f.identity, d), (f.experts + f.identity,)
            for e in range(f.experts):
                gated(f"{q}e{e}", f.ff)
            gated(q + "shared", f.shared)
    return out


def slopes(heads: int) -> torch.Tensor:
    """Bias per position of distance, a geometric series over the heads."""
    return (2.0 ** (-8.0 * (torch.arange(heads, dtype=torch.float64) + 1) / heads)).float()


def build_weights(cfg: ZazilixConfig, get: Callable[[str], torch.Tensor], device) -> Dict[str, torch.Tensor]:
    """``get(name)`` returns a raw tensor; shapes are checked against the configuration."""
    want = raw_shapes(cfg)

    def raw(name):
        t = get(name)
        if tuple(t.shape) != want[name]:
            raise ValueError(f"{name}: shape {tuple(t.shape)} does not fit the configuration ({want[name]})")
        return t

    mat = lambda name: raw(name).to(torch.bfloat16).to(device).contiguous()
    vec = lambda name: raw(name).to(device).float().reshape(-1).contiguous()
    side_by_side = lambda parts: torch.cat([pad(t, (0, 0, 0, -t.shape[0] % 8)) for t in parts], 0)
    w: Dict[str, torch.Tensor] = {"embed.weight": mat("embed"), "pos.weight": mat("pos"), "head.weight": mat("head")}
    w["final.pre"] = torch.cat([torch.ones(cfg.streams, device=device), vec("final.norm")])

    def connections(p, q):
        w[f"{p}hc{q}.pre"] = torch.cat([vec(f"{p}hc{q}.in"), vec(f"{p}norm{q}")])
        w[f"{p}hc{q}.post"] = torch.cat([vec(f"{p}hc{q}.out"), vec(f"{p}hc{q}.mix")])

    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        q = p + "mix."
        connections(p, 1)
        if isinstance(m, MLSTMSpec):
            w[q + "in"] = side_by_side([mat(q + n) for n in "qkvg"])
            w[q + "gates"] = torch.cat([mat(q + "i"), mat(q + "f")], 0)
            w[q + "gates.b"] = torch.cat([vec(q + "i.b"), vec(q + "f.b")])
            w[q + "norm"], w[q + "o"] = vec(q + "norm"), mat(q + "o")
        elif isinstance(m, ParallelSpec):
            a, r = q + "left.", q + "right."
            w[q + "in"] = side_by_side([torch.cat([mat(a + n) for n in "qkv"], 0), mat(r + "q"), mat(r + "v")])
            w[a + "qk.norm"] = torch.cat([vec(a + "q.norm"), vec(a + "k.norm")])
            w[a + "slope"], w[a + "sink"] = slopes(m.left.heads).to(device), torch.zeros(m.left.heads, device=device)
            w[a + "o"], w[r + "o"], w[r + "f"] = mat(a + "o"), mat(r + "o"), mat(r + "f")
            w[r + "f.b"], w[r + "lower"], w[r + "norm"] = vec(r + "f.b"), vec(r + "lower"), vec(r + "norm")
        else:
            inn, inner = mat(q + "in"), m.heads * m.vdim
            w[q + "in"] = side_by_side([inn[:inner], inn[inner:-m.heads]])
            w[q + "dt"] = inn[-m.heads:].contiguous()
            w[q + "conv"] = raw(q + "conv").to(device).float().t().contiguous()
            for n in ("conv.b", "dt_bias", "A_log", "D", "norm"):
                w[q + n] = vec(q + n)
            w[q + "o"] = mat(q + "o")
        f = l.ff
        if f is None:
            continue
        connections(p, 2)
        q = p + "mlp."
        w[q + "router"], w[q + "correction"] = mat(q + "router"), vec(q + "correction")
        w13 = torch.empty(f.experts, 2, f.ff, cfg.hidden_size, dtype=torch.bfloat16, device=device)
        w2 = torch.empty(f.experts, cfg.hidden_size, f.ff, dtype=torch.bfloat16, device=device)
        for e in range(f.experts):
            w13[e, 0], w13[e, 1] = mat(f"{q}e{e}.gate"), mat(f"{q}e{e}.up")
            w2[e] = mat(f"{q}e{e}.down")
        w[q + "w13"], w[q + "w2"] = w13, w2
        w[q + "shared.gu"] = interleave_gate(mat(q + "shared.gate"), mat(q + "shared.up"))
        w[q + "shared.down"] = pad(mat(q + "shared.down"), (0, -f.shared % GATE_BLOCK)).contiguous()
    return w


def load_checkpoint(folder: str, cfg: ZazilixConfig, device) -> Dict[str, torch.Tensor]:
    """Streams a safetensors checkpoint into runtime tensors on ``device``."""
    return build_weights(cfg, tensor_reader(folder), device)


def random_weights(cfg: ZazilixConfig, device, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Random-init weights: matrices of standard deviation 1 / sqrt(fan-in), gains near one, streams that mostly stay themselves,
    recurrences that remember tens to thousands of tokens."""
    shapes, n = raw_shapes(cfg), cfg.streams
    g = torch.Generator(device=device)
    g.manual_seed(seed * 1000003 + 11)

    def draw(name):
        s = shapes[name]
        r = lambda std: torch.randn(s, generator=g, device=device, dtype=torch.float32) * std
        u = lambda lo, hi: torch.rand(s, generator=g, device=device) * (hi - lo) + lo
        if name in ("embed", "pos"):
            t = r(1.0 if name == "embed" else 0.1)
        elif name.endswith((".in", ".out", ".mix")) and ".hc" in name:
            t = torch.eye(n, device=device) * 0.9 + r(0.05) if name.endswith("mix") else r(0.1) + (1.0 / n if name.endswith("in") else 1.0)
        elif name.endswith("A_log"):
            t = u(-2.0, 1.0)
        elif name.endswith("dt_bias"):
            t = r(1.0) - 3.0
        elif name.endswith("lower"):
            t = u(0.0, 0.9)
        elif name.endswith(".f.b"):
            t = r(1.0) + 4.0
        elif name.endswith(".conv"):
            t = r(0.2) + 0.5
        elif name.endswith((".b", "correction")):
            t = r(0.1)
        elif len(s) < 2:
            t = r(0.1) + 1.0
        else:
            t = r(s[-1] ** -0.5)
        return t.to(torch.bfloat16)

    return build_weights(cfg, draw, device)
