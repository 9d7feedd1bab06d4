"""Checkpoint loading for the Sakevik design: raw tensor names -> the tensors its layers run on.

Matrices stay in the checkpoint's bf16 (in 32-bit serving too: the kernels widen them in registers); vectors become fp32.  Merged or
re-laid for the kernels (every part of a merged projection is padded to a multiple of eight rows, so that the column slices of its
result start on 16 bytes):

  * mingru: ``z, x, g -> in``;
  * attention: ``q | k | v`` and ``g`` -> ``qkvg``; the biases of q, k and v -> ``qkv.b``; the two norms -> ``head.norm``; the angles per
    position of keys (``freq``) and values (``vfreq``);
  * latent_attention: the rows of ``q`` sorted into all unrotated and all rotated parts, and ``dkv`` -> ``qc``; ``uk`` transposed per head
    (``uk_t`` [H*R, dim], absorbed into the query), and with an identity beside it that hands the rotated part of a cached row on to
    every head's key (``uk`` [H * (dim + rot), R + rot], for expanded keys);
  * feed-forward: ``gate, up -> gu`` in alternating blocks of 16 rows, its size padded to a multiple of 16 with zeros.
"""
from __future__ import annotations

from typing import Callable, Dict

import torch
from torch.nn.functional import pad

from .buvalix_weight import GATE_BLOCK, interleave_gate
from .layered_config import rotary_frequencies
from .sakevik_config import MinGRUSpec, SakevikConfig, SigmoidAttentionSpec
from .weight import tensor_reader


def raw_shapes(cfg: SakevikConfig) -> Dict[str, tuple]:
    """Names and shapes of the checkpoint's tensors."""
    d = cfg.hidden_size
    out: Dict[str, tuple] = {"embed": (cfg.vocab_size, d), "bigram": (cfg.pairs.buckets + 1, d), "final.norm": (d,),
                             "head": (cfg.vocab_size, d)}
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        q = p + "mix."
        out[p + "norm1"] = (d,)
        if isinstance(m, MinGRUSpec):
            out.update({q + n: (m.width, d) for n in "zxg"})
            out.update({q + "z.b": (m.width,), q + "x.b": (m.width,), q + "o": (d, m.width)})
        elif isinstance(m, SigmoidAttentionSpec):
            for n, rows in (("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
                out[q + n], out[q + n + ".b"] = (rows, d), (rows,)
            out.update({q + "q.norm": (m.dim,), q + "k.norm": (m.dim,), q + "pb": (m.heads,), q + "g": (m.heads, d),
                        q + "o": (d, m.heads * m.vdim), q + "o.b": (d,)})
        else:
            h, r = m.heads, m.kv_rank
            out.update({q + "q": (h * (m.dim + m.rot_dim), d), q + "dkv": (r + m.rot_dim, d), q + "dkv.norm": (r,),
                        q + "uk": (h * m.dim, r), q + "uv": (h * m.vdim, r), q + "o": (d, h * m.vdim)})
        if l.ff is not None:
            out[p + "norm2"] = (d,)
            out[p + "mlp.gate"] = out[p + "mlp.up"] = (l.ff.ff, d)
            out[p + "mlp.down"] = (d, l.ff.ff)
    return out


def build_weights(cfg: SakevikConfig, get: Callable[[str], torch.Tensor], device) -> Dict[str, torch.Tensor]:
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
    w: Dict[str, torch.Tensor] = {"embed.weight": mat("embed"), "pairs.weight": mat("bigram"), "head.weight": mat("head"),
                                  "final.gain": vec("final.norm")}
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        q = p + "mix."
        w[p + "norm1"] = vec(p + "norm1")
        if isinstance(m, MinGRUSpec):
            w[q + "in"] = side_by_side([mat(q + n) for n in "zxg"])
            w[q + "z.b"], w[q + "x.b"] = vec(q + "z.b"), vec(q + "x.b")
        elif isinstance(m, SigmoidAttentionSpec):
            w[q + "qkvg"] = side_by_side([torch.cat([mat(q + n) for n in "qkv"], 0), mat(q + "g")])
            w[q + "qkv.b"] = torch.cat([vec(f"{q}{n}.b") for n in "qkv"])
            w[q + "head.norm"] = torch.stack([vec(q + "q.norm"), vec(q + "k.norm")])
            w[q + "freq"] = rotary_frequencies(m.rot.dims, m.rot.base, m.rot.scaling)[0].to(device)
            w[q + "vfreq"] = rotary_frequencies(m.vdim, m.rot.base)[0].to(device)
            w[q + "wbias"], w[q + "o.b"] = vec(q + "pb"), vec(q + "o.b")
        else:
            h, dim, rot, rank = m.heads, m.dim, m.rot_dim, m.kv_rank
            heads = mat(q + "q").view(h, dim + rot, -1)
            w[q + "qc"] = side_by_side([heads[:, :dim].reshape(h * dim, -1), heads[:, dim:].reshape(h * rot, -1), mat(q + "dkv")])
            w[q + "latent.gain"], w[q + "uv"] = vec(q + "dkv.norm"), mat(q + "uv")
            uk = mat(q + "uk").view(h, dim, rank)
            w[q + "uk_t"] = uk.transpose(1, 2).reshape(-1, dim).contiguous()
            whole = torch.zeros(h, dim + rot, rank + rot, dtype=uk.dtype, device=uk.device)
            whole[:, :dim, :rank] = uk
            whole[:, dim:, rank:] = torch.eye(rot, dtype=uk.dtype, device=uk.device)
            w[q + "uk"] = whole.view(h * (dim + rot), rank + rot)
            w[q + "freq"] = rotary_frequencies(rot, m.rot.base, m.rot.scaling)[0].to(device)
        w[q + "o"] = mat(q + "o")
        if l.ff is not None:
            w[p + "norm2"] = vec(p + "norm2")
            w[p + "mlp.gu"] = interleave_gate(mat(p + "mlp.gate"), mat(p + "mlp.up"))
            w[p + "mlp.down"] = pad(mat(p + "mlp.down"), (0, -l.ff.ff % GATE_BLOCK)).contiguous()
    return w


def load_checkpoint(folder: str, cfg: SakevikConfig, device) -> Dict[str, torch.Tensor]:
    """Streams a safetensors checkpoint into runtime tensors on ``device``."""
    return build_weights(cfg, tensor_reader(folder), device)


def random_weights(cfg: SakevikConfig, device, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Random-init weights: matrices of standard deviation 1 / sqrt(fan-in), gains near one, recurrences that remember tens of tokens,
    attention weights of about a tenth."""
    shapes = raw_shapes(cfg)
    g = torch.Generator(device=device)
    g.manual_seed(seed * 1000003 + 11)

    def draw(name):
        s = shapes[name]
        r = lambda std: torch.randn(s, generator=g, device=device, dtype=torch.float32) * std
        if name in ("embed", "bigram"):
            t = r(1.0)
        elif name.endswith((".z.b", ".pb")):
            t = r(1.0) - 2.5
        elif name.endswith(".b"):
            t = r(0.1)
        elif len(s) == 1:
            t = r(0.1) + 1.0
        else:
            t = r(s[-1] ** -0.5)
        return t.to(torch.bfloat16)

    return build_weights(cfg, draw, device)
