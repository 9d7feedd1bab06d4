"""Python wrappers around the sm_100a kernels of the designs with layer norms around the sub-layers, grouped attention and the
gated delta rule (csrc/residual.cu, grouped_attn.cu, flash_attn.cu, delta.cu, delta_chunk.cu), one function per facade op in
:mod:`minisgl.ops.api`.  Activations are bf16 or fp32."""
from __future__ import annotations

import os

import torch

from . import native as nv
from .cuda import num_sms
from .cuda_layers import KV_ALIGN, SMEM_BYTES, _chunk_plan, _f32, prompt_items, window_span
from .gemm import ACTS, _tma_ok, linear
from .native import F, I
from .tensorcheck import tensors


# --------------------------------------------------------------------------- residual stream
@tensors(x="f32[_,D]", add="?bf16|f32[_,D]", rows="?i64[_]")
def residual_layer_norm(x, eps, dtype, norm, sub, add, rows, keep):
    n, d = x.shape
    y = yw = yb = w = b = out = None
    if sub is not None:
        y, yw, yb = sub
        assert y.shape == (n, d) and y.dtype == torch.float32 and y.is_contiguous()
    assert add is None or add.dtype == dtype
    n_out = n if rows is None else rows.shape[0]
    if norm is not None:
        w, b = norm
        out = torch.empty(n_out, d, dtype=dtype, device=x.device)
    keep = keep and (sub is not None or add is not None)
    nv.call("residual_layer_norm", nv.ptr(x), nv.ptr(rows), nv.ptr(y), nv.ptr(yw), nv.ptr(yb), nv.ptr(add), nv.ptr(w),
            nv.ptr(b), F(eps), I(1 if keep else 0), nv.ptr(out), I(n_out), I(d), _f32(dtype))
    return out


# --------------------------------------------------------------------------- gated feed-forward
GATE_ACTS = {"gelu_tanh": "gelu_gate", "silu": "silu_gate", "clamp": "clamp_gate"}


def gated_linear(h, w, act, block, limit):
    if act not in GATE_ACTS or block != 16:
        raise ValueError(f"no kernel for the gate {act!r} in blocks of {block}")
    if _tma_ok(h, w, h.shape[1]):
        return linear(h, w, act=GATE_ACTS[act], limit=limit)
    gu = linear(h, w)
    t, f = h.shape[0], w.shape[0] // 2
    out = torch.empty(t, f, dtype=h.dtype, device=h.device)
    nv.call("gate_mul", nv.ptr(gu), nv.ptr(out), I(t), I(f), I(ACTS[GATE_ACTS[act]]), F(limit), _f32(h.dtype))
    return out


# --------------------------------------------------------------------------- grouped attention
@tensors(qkv="bf16|f32[T,_]s", bias="?f32[_]", freq="?f32[_]", keys="bf16|f32[R,_]", values="bf16|f32[R,_]", gain="?f32[_]")
def rotate_store(qkv, bias, freq, q_temp, keys, values, fb, heads, kv_heads, dim, vdim, gain, unit_v, eps, v_mul):
    t = qkv.shape[0]
    assert qkv.dtype == keys.dtype == values.dtype and qkv.shape[1] == (heads + kv_heads) * dim + kv_heads * vdim
    assert keys.shape[1] == kv_heads * dim and values.shape[1] == kv_heads * vdim
    assert gain is None or gain.shape[0] == (heads + kv_heads) * dim
    q = torch.empty(t, heads, dim, dtype=qkv.dtype, device=qkv.device)
    coef, every = q_temp if q_temp is not None else (0.0, 0)
    nv.call("rotate_store", nv.ptr(qkv), I(qkv.stride(0)), nv.ptr(bias), nv.ptr(freq), I(0 if freq is None else freq.shape[0]),
            F(coef), I(every), nv.ptr(gain), I(1 if unit_v else 0), F(eps), F(v_mul), nv.ptr(fb.positions), nv.ptr(fb.out_loc),
            nv.ptr(q), nv.ptr(keys), nv.ptr(values), I(t), I(heads), I(kv_heads), I(dim), I(vdim), _f32(qkv.dtype))
    return q


@tensors(qkv="bf16|f32[T,_]s", bias="?f32[_]", gain="?f32[2,_]", freq="?f32[_]", vfreq="?f32[_]", keys="bf16|f32[R,_]",
         values="bf16|f32[R,_]")
def head_store(qkv, bias, gain, eps, freq, mul, vfreq, halves, keys, values, fb, heads, kv_heads, dim, vdim):
    t = qkv.shape[0]
    assert qkv.dtype == keys.dtype == values.dtype and qkv.shape[1] == (heads + kv_heads) * dim + kv_heads * vdim
    assert keys.shape[1] == kv_heads * dim and values.shape[1] == kv_heads * vdim
    assert (gain is None or gain.shape[1] == dim) and (vfreq is None or 2 * vfreq.shape[0] == vdim)
    q = torch.empty(t, heads, dim, dtype=qkv.dtype, device=qkv.device)
    turn = None if vfreq is None else torch.empty(t, vdim // 2, 2, dtype=torch.float32, device=qkv.device)
    nv.call("head_store", nv.ptr(qkv), I(qkv.stride(0)), nv.ptr(bias), nv.ptr(gain), F(eps), nv.ptr(freq),
            I(0 if freq is None else freq.shape[0]), I(1 if halves else 0), F(mul), nv.ptr(vfreq), nv.ptr(turn),
            nv.ptr(fb.positions), nv.ptr(fb.out_loc), nv.ptr(q), nv.ptr(keys), nv.ptr(values), I(t), I(heads), I(kv_heads), I(dim),
            I(vdim), _f32(qkv.dtype))
    return q, turn


# Portions of at least FLASH_MIN tokens run on the prompt kernel (csrc/flash_attn.cu), shorter ones and single tokens on
# grouped_attn.cu.  MINISGL_GROUPED_PREFILL: auto, flash (every portion that the kernel takes) or rows (none).
GROUPED_PREFILL = os.environ.get("MINISGL_GROUPED_PREFILL", "auto")
FLASH_MIN = 64
FLASH_BYTES = 4 << 30           # bound of the gathered keys and values of one call


def row_tile(rows_per_request: int) -> int:
    return 16 if rows_per_request <= 16 else 32 if rows_per_request <= 32 else 64


def _split_keys(tiles: int, kv_heads: int, m: int, width: int, max_context: int, sms: int) -> int:
    """Ways to split the keys: pays while the row tiles alone leave SMs idle and a tile has several key tiles."""
    p = 64 if width <= 64 else 128 if width <= 128 else 256
    smem = m * p * 2 + 4 * 64 * p * 2 + m * 68 * 4 + m * 64 * 2 + 20 * m
    ctas = sms * max(1, min(SMEM_BYTES // smem, 4))
    return max(1, min(ctas // max(tiles * kv_heads, 1), -(-max_context // 128), 32))


def _pieces(fb, chunk: int, window: int):
    """The portions of a forward, cut where a chunk of keys ends: (queries, keys up to the last one's own, slot, first key).  With a
    window the first key is the first that any of them sees."""
    for n, s, slot in zip(fb.seg_lens, fb.seg_ends, fb.seg_slots):
        if window:
            key0 = max(0, s - n - window + 1)
            yield n, s - key0, slot, key0
            continue
        at, size = s - n, chunk or s
        while at < s:
            key0 = at // size * size
            end = min(key0 + size, s)
            yield end - at, end - key0, slot, key0
            at = end


def _prefill_plan(fb, device, group: int, flash_ok: bool, chunk: int, window: int):
    """How the requests of a prefill forward are spread over the two kernels; the same for all layers with this many query
    heads to a key head and this chunk size or window: (flash requests [n, 4], flash items [m, 5], n, m, gathered rows, row tiles [k, 2],
    k, rows per tile, longest context among the row tiles)."""
    plans = fb.__dict__.setdefault("grouped_plans", {})
    key = (group, flash_ok, GROUPED_PREFILL, FLASH_MIN, chunk, window)
    if key in plans:
        return plans[key]
    least = 1 if GROUPED_PREFILL == "flash" else FLASH_MIN
    pieces = list(_pieces(fb, chunk, window))
    flash = [flash_ok and n >= least for n, _, _, _ in pieces]
    few = [p[0] for p, f in zip(pieces, flash) if not f]
    m = row_tile(max(few) * group) if few else 16
    reqs, items, tiles, at, row, longest = [], [], [], 0, 0, 1
    for (n, s, slot, key0), f in zip(pieces, flash):
        if f:
            reqs.append((slot, s, at, key0))
            items += prompt_items(row, n, s, at, window)
            at += -(-s // KV_ALIGN) * KV_ALIGN
        else:
            tiles += [(r, min(r + m, (row + n) * group)) for r in range(row * group, (row + n) * group, m)]
            longest = max(longest, min(s, window + m // group) if window else s)
        row += n
    items.sort(key=lambda i: -i[4])                   # the longest first
    host = torch.tensor([v for t in (*reqs, *items, *tiles) for v in t], dtype=torch.int32).pin_memory()
    dev = host.to(device, non_blocking=True)
    a, b = 4 * len(reqs), 4 * len(reqs) + 5 * len(items)
    plans[key] = (dev[:a], dev[a:b], len(reqs), len(items), at, dev[b:], len(tiles), m, longest)
    return plans[key]


@tensors(q="bf16|f32[T,H,D]", keys="bf16|f32[R,_]", values="bf16|f32[R,_]", sink="?f32[H]", rel="?f32[H,_]", slope="?f32[H]",
         wbias="?f32[H]", turn="?f32[T,_,2]", gate="?bf16|f32[T,H]s")
def grouped_attention(q, keys, values, fb, kv_heads, scale, softcap, sink, rel, slope, chunk, window, wbias, turn, gate):
    t, heads, dim = q.shape
    group, kw, vw = heads // kv_heads, keys.shape[1], values.shape[1]
    vdim = vw // kv_heads
    assert q.dtype == keys.dtype == values.dtype and kw == kv_heads * dim and (gate is None or gate.dtype == q.dtype)
    assert turn is None or 2 * turn.shape[1] == vdim
    ends = (nv.ptr(wbias), nv.ptr(turn), nv.ptr(gate), I(0 if gate is None else gate.stride(0)))
    out = torch.empty(t, heads * vdim, dtype=q.dtype, device=q.device)
    pt, n_rel = fb.page_table, 0 if rel is None else rel.shape[1]
    even = q.dtype == torch.bfloat16 and dim % 8 == 0 and vdim % 8 == 0
    tiles, n_tiles, m, longest = None, 0, 0, min(fb.max_context, chunk) if chunk else window_span(fb, window)
    if even and fb.seg_lens is not None:
        ctx = sum(-(-s // KV_ALIGN) * KV_ALIGN for s in fb.seg_ends)
        flash_ok = max(dim, vdim) <= 128 and GROUPED_PREFILL != "rows" and 2 * ctx * (kw + vw) <= FLASH_BYTES
        flash_ok = flash_ok and not (slope is not None and (softcap or rel is not None)) and (turn is None or vdim % 32 == 0)
        flash_ok = flash_ok and not (wbias is not None and (softcap or rel is not None or slope is not None))
        reqs, items, n_reqs, n_items, rows, tiles, n_tiles, m, longest = _prefill_plan(fb, q.device, group, flash_ok, chunk,
                                                                                                  window)
        if n_items:
            ck = torch.empty(rows, kw, dtype=q.dtype, device=q.device)
            cv = torch.empty(vw, rows, dtype=q.dtype, device=q.device)
            nv.call("kv_gather", nv.ptr(keys), nv.ptr(values), nv.ptr(ck), nv.ptr(cv), nv.ptr(reqs), I(n_reqs), I(rows),
                    nv.ptr(pt), I(pt.stride(0)), I(kw), I(vw))
            nv.call("flash_attention", nv.ptr(q), I(heads * dim), nv.ptr(ck), nv.ptr(cv), nv.ptr(out), nv.ptr(items),
                    I(n_items), I(t), I(rows), I(heads), I(kv_heads), I(dim), I(vdim), F(scale), F(softcap), nv.ptr(sink),
                    nv.ptr(rel), I(n_rel), nv.ptr(slope), ends[0], I(window), *ends[1:])
        if n_tiles == 0:
            return out
    elif even:
        m = row_tile(group)
        n_tiles = t * -(-group // m)
    if max(dim, vdim) > 256:
        if tiles is not None and n_tiles:
            tiles = None                # the one-warp-per-row kernel takes every token
        m = 0
    nsplit, acc, ml = 1, None, None
    if m:
        nsplit = _split_keys(n_tiles, kv_heads, m, max(dim, vdim), longest, num_sms(q.device))
        if nsplit > 1 or turn is not None or gate is not None:
            acc = torch.empty(t * heads, nsplit, vdim, dtype=torch.float32, device=q.device)
            ml = torch.empty(t * heads, nsplit, 2, dtype=torch.float32, device=q.device)
    nv.call("grouped_attention", nv.ptr(q), nv.ptr(keys), nv.ptr(values), nv.ptr(out), nv.ptr(fb.slots), nv.ptr(fb.positions),
            nv.ptr(pt), I(pt.stride(0)), nv.ptr(tiles), I(n_tiles), nv.ptr(fb.num_valid), I(t), I(kv_heads), I(group), I(dim),
            I(vdim), F(scale), F(softcap), nv.ptr(sink), nv.ptr(rel), I(n_rel), nv.ptr(slope), I(chunk), I(window), *ends, I(m),
            I(nsplit), nv.ptr(acc), nv.ptr(ml), _f32(q.dtype))
    return out


# --------------------------------------------------------------------------- gated delta rule
def _columns(heads: int, kv_heads: int, dim: int, vdim: int):
    up = -(-kv_heads * dim // 8) * 8
    return up, 2 * up                     # first columns of k and of v in the merged projection


@tensors(p="bf16|f32[T,_]", taps="f32[N,C]", before="bf16|f32[_,_,C]")
def conv_unit(p, taps, before, fb, heads, kv_heads, dim, vdim):
    t, qk = p.shape[0], kv_heads * dim
    at_k, at_v = _columns(heads, kv_heads, dim, vdim)
    assert before.dtype == p.dtype and before.shape[1] == taps.shape[0] - 1 and taps.shape[1] == 2 * qk + heads * vdim
    q = torch.empty(t, qk, dtype=torch.float32, device=p.device)
    k = torch.empty_like(q)
    v = torch.empty(t, heads * vdim, dtype=p.dtype, device=p.device)
    nv.call("conv_unit", nv.ptr(p), I(p.stride(0)), I(at_k), I(at_v), nv.ptr(taps), I(taps.shape[0]), nv.ptr(before),
            nv.ptr(fb.slots), nv.ptr(fb.positions), nv.ptr(q), nv.ptr(k), nv.ptr(v), I(t), I(heads), I(kv_heads), I(dim),
            I(vdim), _f32(p.dtype))
    return q, k, v


# Portions of at least DELTA_CHUNK_MIN tokens run the recurrence in chunks (csrc/delta_chunk.cu).  In 32-bit serving it stays
# token by token: decays are then products of the decays themselves, not exponentials of sums.  DELTA_CHUNKED overrides.
DELTA_CHUNKED = None
DELTA_CHUNK_MIN = 64


@tensors(q="f32[T,_]", k="f32[T,_]", v="bf16|f32[T,V]", rate="f32[T,N]", dt_bias="f32[N]", a_log="f32[H]", p="bf16|f32[T,_]",
         gate="bf16|f32[T,V]", gain="f32[_]", state="f32[S,H,_,_]", before="bf16|f32[S,_,_]")
def delta_rule(q, k, v, rate, dt_bias, a_log, p, at_b, gate, gain, eps, state, before, fb, heads, kv_heads):
    t, dim, vdim = q.shape[0], state.shape[2], state.shape[3]
    assert v.dtype == gate.dtype == p.dtype == before.dtype and rate.shape[1] == heads * dim
    at_k, at_v = _columns(heads, kv_heads, dim, vdim)
    taps, f32 = before.shape[1] + 1, dict(dtype=torch.float32, device=q.device)
    y = torch.empty_like(v)
    chunked = DELTA_CHUNKED if DELTA_CHUNKED is not None else p.dtype == torch.bfloat16
    chunked = chunked and dim % 4 == 0 and vdim % 4 == 0 and dim <= 128
    norm = lambda raw: nv.call("head_norm_gate", nv.ptr(raw), nv.ptr(gate), nv.ptr(gain), F(eps), nv.ptr(y), I(t), I(heads),
                               I(vdim), _f32(p.dtype))
    if chunked and fb.seg_lens is not None and max(fb.seg_lens) >= DELTA_CHUNK_MIN:
        chunks, segs, n, n_segs = _chunk_plan(fb, q.device)
        raw = torch.empty(t, heads * vdim, **f32)
        w, kr, qd = (torch.empty(n, heads, 32, dim, **f32) for _ in range(3))
        u0, b, decay = (torch.empty(n, heads, *s, **f32) for s in ((32, vdim), (32, 32), (dim,)))
        nv.call("delta_chunked", nv.ptr(p), I(p.stride(0)), I(at_k), I(at_v), I(at_b), I(taps), nv.ptr(q), nv.ptr(k),
                nv.ptr(v), nv.ptr(rate), nv.ptr(dt_bias), nv.ptr(a_log), nv.ptr(state), nv.ptr(before), nv.ptr(raw),
                nv.ptr(fb.positions), nv.ptr(fb.seg_off), nv.ptr(chunks), I(n), nv.ptr(segs), I(n_segs), nv.ptr(w),
                nv.ptr(kr), nv.ptr(qd), nv.ptr(u0), nv.ptr(b), nv.ptr(decay), I(heads), I(kv_heads), I(dim), I(vdim),
                _f32(p.dtype))
        norm(raw)
        return y
    vb = 64 if vdim <= 64 or dim > 128 else 128
    raw = torch.empty(t, heads * vdim, **f32) if vdim > vb else None
    segs = t if fb.seg_off is None else fb.seg_off.shape[0] - 1
    nv.call("delta_scan", nv.ptr(p), I(p.stride(0)), I(at_k), I(at_v), I(at_b), I(taps), nv.ptr(q), nv.ptr(k), nv.ptr(v),
            nv.ptr(rate), nv.ptr(dt_bias), nv.ptr(a_log), nv.ptr(gate), nv.ptr(gain), F(eps), nv.ptr(state), nv.ptr(before),
            nv.ptr(raw), nv.ptr(fb.slots), nv.ptr(fb.positions), nv.ptr(fb.seg_off), I(segs),
            nv.ptr(fb.num_valid if fb.seg_off is None else None), I(heads), I(kv_heads), I(dim), I(vdim), I(vb), nv.ptr(y),
            _f32(p.dtype))
    if raw is not None:
        norm(raw)
    return y
