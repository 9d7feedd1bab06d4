"""Python wrappers around the sm_100a kernels of gated linear attention (csrc/gla.cu, gla_chunk.cu), one function per facade op in
:mod:`minisgl.ops.api`.  Activations are bf16 or fp32."""
from __future__ import annotations

import torch

from . import native as nv
from .cuda_layers import _chunk_plan, _f32
from .native import F, I
from .tensorcheck import tensors

MODES = {"given": 0, "step": 1, "forget": 2}
CONV_SPAN = 16           # tokens per tile of the short convolution

# Portions of at least GLA_CHUNK_MIN tokens run the recurrence in chunks (csrc/gla_chunk.cu).  In 32-bit serving it stays token by
# token: decays are then products of the decays themselves, not exponentials of sums.  GLA_CHUNKED = False turns chunks off.
GLA_CHUNKED = True
GLA_CHUNK, GLA_CHUNK_MIN = 64, 64


def _segments(fb, rows: int):
    """(segment offsets or None, segments, valid segments or None)."""
    if fb.seg_off is None:
        return None, rows, fb.num_valid
    return fb.seg_off, fb.seg_off.shape[0] - 1, None


@tensors(z="f32[T,_]", bias="f32[_]", top="f32[_,H]")
def mlstm_gates(z, bias, cap, top, fb):
    t, heads = z.shape[0], top.shape[1]
    assert z.shape[1] == bias.shape[0] == 2 * heads
    out = torch.empty(3, t, heads, dtype=torch.float32, device=z.device)
    off, segs, valid = _segments(fb, t)
    nv.call("mlstm_gates", nv.ptr(z), nv.ptr(bias), F(cap), nv.ptr(top), nv.ptr(out[0]), nv.ptr(out[1]), nv.ptr(out[2]),
            nv.ptr(fb.slots), nv.ptr(fb.positions), nv.ptr(off), I(segs), nv.ptr(valid), I(heads),
            I(max(fb.seg_lens) if fb.seg_lens is not None else 1))
    return out[0], out[1], out[2]


def _conv_tiles(fb, device, span: int):
    """[tiles, 2]: segment and first token within it, every ``span`` tokens; the same for all layers."""
    plans = fb.__dict__.setdefault("conv_plans", {})
    if span not in plans:
        host = torch.tensor([(s, o) for s, n in enumerate(fb.seg_lens) for o in range(0, n, span)], dtype=torch.int32)
        plans[span] = host.pin_memory().to(device, non_blocking=True)
    return plans[span]


@tensors(p="bf16|f32[T,C]s", taps="f32[N,C]", bias="f32[C]", before="bf16|f32[_,_,C]")
def causal_conv(p, taps, bias, before, fb):
    t, c = p.shape
    n = taps.shape[0]
    assert before.dtype == p.dtype and before.shape[1] == n - 1
    out = torch.empty(t, c, dtype=p.dtype, device=p.device)
    tiles = _conv_tiles(fb, p.device, CONV_SPAN) if fb.seg_lens is not None else None
    for lo in range(0, t if tiles is None else tiles.shape[0], 65535):
        part = None if tiles is None else tiles[lo:lo + 65535]
        nv.call("causal_conv", nv.ptr(p), I(p.stride(0)), nv.ptr(taps), I(n), nv.ptr(bias), nv.ptr(before), nv.ptr(out), I(c),
                nv.ptr(fb.slots), nv.ptr(fb.positions), nv.ptr(fb.seg_off), nv.ptr(part), I(t if part is None else len(part)),
                I(CONV_SPAN), nv.ptr(fb.num_valid if part is None else None), _f32(p.dtype))
    return out


@tensors(q="bf16|f32[T,_]s", k="?bf16|f32[T,_]s", v="bf16|f32[T,_]s", state="f32[_,H,_,_]")
def gla(kind, q, k, v, gates, state, fb, heads, groups, q_mul):
    t, (d, ew) = v.shape[0], state.shape[2:]
    e = v.shape[1] // heads
    assert state.shape[1] == heads and q.shape[1] == groups * d and (k is None) == (kind == "forget")
    assert q.dtype == v.dtype and (k is None or (k.dtype == v.dtype and k.shape[1] == groups * d))
    raw, fac, bias, par = (gates[0], gates[1], None, None) if kind == "given" else (gates[0], None, gates[1], gates[2])
    rows = heads * d if kind == "forget" else heads
    assert raw.shape == (t, rows) and all(g.is_contiguous() and g.dtype == torch.float32 for g in gates)
    out = torch.empty(t, heads, ew, dtype=torch.float32, device=v.device)
    ldk = 0 if k is None else k.stride(0)
    common = (I(MODES[kind]), nv.ptr(q), I(q.stride(0)), nv.ptr(k), I(ldk), nv.ptr(v), I(v.stride(0)), nv.ptr(raw), nv.ptr(fac),
              nv.ptr(bias), nv.ptr(par), F(q_mul), nv.ptr(state), nv.ptr(out))
    sizes = (I(heads), I(heads // groups), I(d), I(e), I(ew))
    even = d % 8 == 0 and e % 8 == 0 and d <= 128 and all(x is None or (x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0)
                                                            for x in (q, k, v))
    if GLA_CHUNKED and v.dtype == torch.bfloat16 and even and fb.seg_lens is not None and max(fb.seg_lens) >= GLA_CHUNK_MIN:
        chunks, segs, n, n_segs = _chunk_plan(fb, v.device, GLA_CHUNK)
        us = torch.empty(n, heads, d, ew, dtype=torch.float32, device=v.device)
        decay = torch.empty(n, rows, dtype=torch.float32, device=v.device)
        nv.call("gla_chunked", *common, nv.ptr(fb.positions), nv.ptr(chunks), I(n), nv.ptr(segs), I(n_segs), nv.ptr(us),
                nv.ptr(decay), *sizes)
        return out
    off, segs, valid = _segments(fb, t)
    nv.call("gla_scan", *common, nv.ptr(fb.slots), nv.ptr(fb.positions), nv.ptr(off), I(segs), nv.ptr(valid), *sizes,
            _f32(v.dtype))
    return out


@tensors(o="f32[T,H,_]", gain="f32[_]", gate="?bf16|f32[T,_]s", floor="?f32[T,H]")
def norm_heads(o, e, gain, eps, dtype, gate, floor, mul):
    t, heads, ew = o.shape
    assert gain.shape[0] in (e, heads * e) and (gate is None or gate.dtype == dtype) and (floor is None or ew > e)
    y = torch.empty(t, heads * e, dtype=dtype, device=o.device)
    per_head = gain.shape[0] == heads * e
    nv.call("gla_norm_heads", nv.ptr(o), nv.ptr(floor), nv.ptr(gate), I(0 if gate is None else gate.stride(0)), nv.ptr(gain),
            I(1 if per_head else 0), F(eps), F(mul), nv.ptr(y), I(heads * e), I(t), I(heads), I(e), I(ew), _f32(dtype))
    return y


@tensors(o="f32[T,H,_]", skip="f32[H]", x="bf16|f32[T,N]s", z="bf16|f32[T,N]s", gain="f32[N]")
def norm_groups(o, skip, x, z, gain, groups, eps):
    t, heads, ew = o.shape
    assert x.dtype == z.dtype
    y = torch.empty(t, x.shape[1], dtype=x.dtype, device=o.device)
    nv.call("gla_norm_groups", nv.ptr(o), nv.ptr(skip), nv.ptr(x), I(x.stride(0)), nv.ptr(z), I(z.stride(0)), nv.ptr(gain),
            I(groups), F(eps), nv.ptr(y), I(t), I(heads), I(x.shape[1] // heads), I(ew), _f32(x.dtype))
    return y
