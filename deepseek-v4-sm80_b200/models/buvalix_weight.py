"""Checkpoint loading for the Buvalix design: raw tensor names -> the tensors its layers run on.

Matrices stay in the checkpoint's bf16 (in 32-bit serving too: the kernels widen them in registers); vectors become fp32.
Merged or re-laid for the kernels:

  * attention: ``q, k, v -> qkv`` (one projection) with ``qkv.b``; the rotation's frequencies ``freq``; the distance table
    ``rel`` [buckets, H] spread out to one value per distance, ``rel`` [H, distances];
  * channel_delta: ``q, k, v, a1, g1, b -> in`` (one projection, every part padded to a multiple of eight rows so that the
    column slices of its result start on 16 bytes); the three convolutions as one [taps, channels] table;
  * feed-forward: ``gate, up -> gu`` in alternating blocks of 16 rows (the projection's epilogue pairs them), the feed-forward
    size padded to a multiple of 16 with zeros.
"""
from __future__ import annotations

import math
from typing import Callable, Dict

import torch

from .buvalix_config import BuvalixConfig, ChannelDeltaSpec
from .weight import tensor_reader

FREE = -1     # a size that only the tensors give
GATE_BLOCK = 16
DELTA_PARTS = ("q", "k", "v", "a1", "g1", "b")     # the merged input projection of a channel_delta layer, in order


def raw_shapes(cfg: BuvalixConfig) -> Dict[str, tuple]:
    """Names and shapes of the checkpoint's tensors."""
    d = cfg.hidden_size
    out: Dict[str, tuple] = {"embed": (cfg.vocab_size, d), "head": (cfg.vocab_size, d)}

    def norm(name):
        out[name] = out[name + ".b"] = (d,)

    norm("final.norm")
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        q = p + "mix."
        norm(p + "norm1")
        norm(p + "norm1b")
        h, g = m.heads, m.kv_heads
        if isinstance(m, ChannelDeltaSpec):
            rows = {"q": g * m.dim, "k": g * m.dim, "v": h * m.vdim}
            out.update({q + n: (r, d) for n, r in rows.items()})
            out.update({q + n + ".conv": (r, m.conv) for n, r in rows.items()})
            out.update({q + "b": (h, d), q + "A_log": (h,), q + "norm": (m.vdim,), q + "dt_bias": (h * m.dim,),
                        q + "a1": (FREE, d), q + "a2": (h * m.dim, FREE), q + "g1": (FREE, d), q + "g2": (h * m.vdim, FREE)})
        else:
            rows = {"q": h * m.dim, "k": g * m.dim, "v": g * m.vdim}
            out.update({q + n: (r, d) for n, r in rows.items()})
            if m.bias:
                out.update({q + n + ".b": (r,) for n, r in rows.items()})
            if m.sink:
                out[q + "sink"] = (h,)
            if m.bias_max:
                out[q + "rel"] = (FREE, h)
        out[q + "o"] = (d, h * m.vdim)
        if l.ff is not None:
            norm(p + "norm2")
            norm(p + "norm2b")
            out[p + "mlp.gate"] = out[p + "mlp.up"] = (l.ff.ff, d)
            out[p + "mlp.down"] = (d, l.ff.ff)
    return out


def spread_buckets(rel: torch.Tensor, limit: int) -> torch.Tensor:
    """[buckets, H] -> [H, distances]: the bias of every distance, the last entry standing for all that are further.  The
    first half of the buckets holds one distance each, the rest grow evenly in the logarithm up to ``limit``."""
    rows = rel.shape[0]
    half = rows // 2

    def bucket(n):
        if n < half:
            return n
        if limit <= half or half == 0:
            return rows - 1
        return min(rows - 1, half + math.floor(math.log(n / half) / math.log(limit / half) * (rows - half)))

    idx = [bucket(n) for n in range(max(limit, half) + 1)]
    while len(idx) > 1 and idx[-2] == idx[-1]:
        idx.pop()
    return rel.float()[idx].t().contiguous()


def interleave_gate(gate: torch.Tensor, up: torch.Tensor, block: int = GATE_BLOCK) -> torch.Tensor:
    """[F, D] x 2 -> [2 F', D]: blocks of ``block`` gate rows and the ``block`` matching up rows, zero rows at the end."""
    f, d = gate.shape
    pad = -f % block
    parts = [torch.nn.functional.pad(t, (0, 0, 0, pad)).view(-1, block, d) for t in (gate, up)]
    return torch.stack(parts, 1).reshape(-1, d).contiguous()


def build_weights(cfg: BuvalixConfig, get: Callable[[str], torch.Tensor], device) -> Dict[str, torch.Tensor]:
    """``get(name)`` returns a raw tensor; shapes are checked against the configuration."""
    want = raw_shapes(cfg)

    def raw(name):
        t, shape = get(name), want[name]
        if t.dim() != len(shape) or any(a != b for a, b in zip(t.shape, shape) if b != FREE):
            raise ValueError(f"{name}: shape {tuple(t.shape)} does not fit the configuration ({shape})")
        return t

    mat = lambda name: raw(name).to(torch.bfloat16).to(device).contiguous()
    vec = lambda name: raw(name).to(device).float().reshape(-1).contiguous()
    w: Dict[str, torch.Tensor] = {"embed.weight": mat("embed"), "head.weight": mat("head")}

    def norm(name):
        w[name + ".w"], w[name + ".b"] = vec(name), vec(name + ".b")

    norm("final.norm")
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        q = p + "mix."
        norm(p + "norm1")
        norm(p + "norm1b")
        if isinstance(m, ChannelDeltaSpec):
            parts = {n: mat(q + n) for n in DELTA_PARTS}
            a2, g2 = mat(q + "a2"), mat(q + "g2")
            for n, second in (("a1", a2), ("g1", g2)):
                if parts[n].shape[0] != second.shape[1]:
                    raise ValueError(f"{q}{n}: {parts[n].shape[0]} rows feed {second.shape[1]} columns")
            pad8 = lambda t: torch.nn.functional.pad(t, (0, 0, 0, -t.shape[0] % 8))
            w[q + "in"] = torch.cat([pad8(parts[n]) for n in DELTA_PARTS], 0)
            w[q + "a2"], w[q + "g2"] = a2, g2
            taps = torch.cat([raw(q + n + ".conv").to(device).float() for n in "qkv"], 0)
            w[q + "conv"] = taps.t().contiguous()
            w[q + "A_log"], w[q + "dt_bias"], w[q + "norm"] = vec(q + "A_log"), vec(q + "dt_bias"), vec(q + "norm")
        else:
            w[q + "qkv"] = torch.cat([mat(q + n) for n in "qkv"], 0)
            if m.bias:
                w[q + "qkv.b"] = torch.cat([vec(f"{q}{n}.b") for n in "qkv"])
            if m.rot is not None:
                i2 = torch.arange(m.rot.dims // 2, dtype=torch.float64)
                w[q + "freq"] = (m.rot.base ** (-2.0 * i2 / max(m.rot.dims, 1))).float().to(device)
            if m.sink:
                w[q + "sink"] = vec(q + "sink")
            if m.bias_max:
                w[q + "rel"] = spread_buckets(raw(q + "rel"), m.bias_max).to(device)
        w[q + "o"] = mat(q + "o")
        if l.ff is not None:
            norm(p + "norm2")
            norm(p + "norm2b")
            w[p + "mlp.gu"] = interleave_gate(mat(p + "mlp.gate"), mat(p + "mlp.up"))
            w[p + "mlp.down"] = torch.nn.functional.pad(mat(p + "mlp.down"), (0, -l.ff.ff % GATE_BLOCK)).contiguous()
    return w


def load_checkpoint(folder: str, cfg: BuvalixConfig, device) -> Dict[str, torch.Tensor]:
    """Streams a safetensors checkpoint into runtime tensors on ``device``."""
    return build_weights(cfg, tensor_reader(folder), device)


def random_weights(cfg: BuvalixConfig, device, seed: int = 0, rank: int = 128, buckets: int = 32) -> Dict[str, torch.Tensor]:
    """Random-init weights: matrices of standard deviation 1 / sqrt(fan-in), gains near one, decays of about 0.8 to 0.999 per
    token.  rank: inner size of the decay and gate projections."""
    shapes = raw_shapes(cfg)
    g = torch.Generator(device=device)
    g.manual_seed(seed * 1000003 + 11)

    def draw(name):
        s = tuple((buckets if name.endswith(".rel") else rank) if n == FREE else n for n in shapes[name])
        r = lambda std: torch.randn(*s, generator=g, device=device, dtype=torch.float32) * std
        if name == "embed":
            t = r(1.0)
        elif name.endswith("A_log"):
            t = torch.rand(*s, generator=g, device=device) * 2.0 - 3.0
        elif name.endswith("dt_bias"):
            t = r(0.5) - 1.0
        elif name.endswith((".sink", ".rel")):
            t = r(0.5)
        elif name.endswith(".conv"):
            t = r(0.2) + 0.5
        elif name.endswith(".b") and len(s) == 1:
            t = r(0.1)
        elif len(s) == 1:
            t = r(0.1) + 1.0
        else:
            t = r(s[-1] ** -0.5)
        return t.to(torch.bfloat16)

    return build_weights(cfg, draw, device)
