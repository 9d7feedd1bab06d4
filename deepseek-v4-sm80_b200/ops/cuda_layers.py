"""Python wrappers around the sm_100a kernels of the layered models (csrc/residual.cu, latent_attn.cu, wkv.cu,
moe_bf16.cu, gemm_simt.cu), one function per facade op in :mod:`minisgl.ops.api`.  Activations are bf16 or fp32."""
from __future__ import annotations

import torch

from . import native as nv
from .cuda import num_sms
from .gemm import _tma_ok, gemm_bf16_partials, linear
from .native import F, I, L
from .tensorcheck import tensors

SMEM_BYTES = 227 * 1024


def _f32(dtype) -> I:
    return I(1 if dtype == torch.float32 else 0)


# --------------------------------------------------------------------------- residual stream
@tensors(ids="i32[T]", weight="bf16[_,_]", feedback="?i32[_]", slots="?i32[T]")
def embed_residual(ids, weight, dtype, feedback=None, slots=None, want_act=False):
    t, d = ids.shape[0], weight.shape[1]
    x = torch.empty(t, d, dtype=torch.float32, device=ids.device)
    act = torch.empty(t, d, dtype=dtype, device=ids.device) if want_act else None
    nv.call("embed_residual", nv.ptr(ids), nv.ptr(feedback), nv.ptr(slots), nv.ptr(weight), nv.ptr(x), nv.ptr(act),
            I(t), I(d), _f32(dtype))
    return x, act


@tensors(x="f32[_,D]", gain="?f32[D]", rows="?i64[_]", add="?f32[_,D]", add2="?f32[_,D]", vec="?f32[D]")
def residual_norm(x, gain, eps, dtype, mul=1.0, rows=None, add=None, add2=None, vec=None, experts=None, cast=False):
    n, d = x.shape
    erows = wts = idx = None
    topk = 0
    if experts is not None:
        erows, wts, idx = experts
        topk = idx.shape[1]
        assert erows.dtype == dtype and erows.shape == (n * topk, d) and erows.is_contiguous()
    n_out = n if rows is None else rows.shape[0]
    out = torch.empty(n_out, d, dtype=dtype, device=x.device) if gain is not None or cast else None
    nv.call("residual_norm", nv.ptr(x), nv.ptr(rows), nv.ptr(add), nv.ptr(add2), nv.ptr(vec), nv.ptr(erows),
            nv.ptr(wts), nv.ptr(idx), I(topk), nv.ptr(gain), F(eps), F(mul), nv.ptr(out), I(n_out), I(d), _f32(dtype))
    return out


# --------------------------------------------------------------------------- mixture of experts
@tensors(h="bf16|f32[T,D]", weight="bf16[E,D]", bias="f32[E]", num_valid="?i32[1]")
def route_topk(h, weight, bias, top, num_valid=None):
    t, e = h.shape[0], weight.shape[0]
    if _tma_ok(h, weight, h.shape[1]):
        scores = gemm_bf16_partials(h, weight)      # [S, T, E]; the selection kernel adds the splits
    else:
        scores = linear(h, weight, out_dtype=torch.float32)[None]
    idx = torch.empty(t, top, dtype=torch.int32, device=h.device)
    wts = torch.empty(t, top, dtype=torch.float32, device=h.device)
    nv.call("moe_topk", nv.ptr(scores), nv.ptr(bias), nv.ptr(None), nv.ptr(None), nv.ptr(num_valid), nv.ptr(idx),
            nv.ptr(wts), I(t), I(e), I(top), F(1.0), I(3), I(scores.shape[0]), L(scores.stride(0)))
    return idx, wts


def expert_route_tile(routes: int, experts: int) -> int:
    """Routes per tile of the bf16 grouped GEMM: wide enough that an expert's routes rarely need a second tile (which
    streams the expert's weights again), no wider."""
    avg = routes / max(experts, 1)
    return 16 if avg <= 12 else 32 if avg <= 28 else 64 if avg <= 96 else 128


@tensors(h="bf16|f32[T,D]", idx="i32[T,K]", wts="f32[T,K]", w13="bf16[E,2,F,D]", w2="bf16[E,D,F]")
def gated_experts(h, idx, wts, w13, w2):
    t, d = h.shape
    e, _, f, _ = w13.shape
    top = idx.shape[1]
    routes = t * top
    mma = h.dtype == torch.bfloat16 and d % 8 == 0 and f % 8 == 0
    nt = expert_route_tile(routes, e) if mma else 64
    max_tiles = min(e, routes) + routes // nt + 1
    plan = torch.empty(4 + 3 * max_tiles + 3 * routes, dtype=torch.int32, device=h.device)
    nv.call("moe_plan", nv.ptr(idx), nv.ptr(wts), I(routes), I(e), I(0), I(nt), nv.ptr(plan), I(max_tiles))
    new = lambda n: torch.empty(routes, n, dtype=h.dtype, device=h.device)
    act, rows = new(f), new(d)
    if mma:
        xs = new(d)
        nv.call("moe_gather_rows", nv.ptr(h), nv.ptr(xs), nv.ptr(plan), I(routes), I(max_tiles), I(top), I(d))
        nv.call("moe_bf16_gemm", I(1), I(nt), nv.ptr(w13), nv.ptr(xs), nv.ptr(plan), I(routes), I(max_tiles),
                nv.ptr(act), I(e), I(f), I(d))
        nv.call("moe_bf16_gemm", I(2), I(nt), nv.ptr(w2), nv.ptr(act), nv.ptr(plan), I(routes), I(max_tiles),
                nv.ptr(rows), I(e), I(d), I(f))
        return rows
    gu = new(2 * f)
    nv.call("moe_gemm_simt", nv.ptr(h), nv.ptr(w13), nv.ptr(gu), nv.ptr(plan), I(routes), I(max_tiles), I(e), I(2 * f),
            I(d), I(top), _f32(h.dtype))
    nv.call("silu_mul", nv.ptr(gu), nv.ptr(act), I(routes), I(f), _f32(h.dtype))
    nv.call("moe_gemm_simt", nv.ptr(act), nv.ptr(w2), nv.ptr(rows), nv.ptr(plan), I(routes), I(max_tiles), I(e), I(d),
            I(f), I(1), _f32(h.dtype))
    return rows


# --------------------------------------------------------------------------- latent attention
@tensors(x="bf16|f32[_,R]s", gain="f32[R]", cache="bf16|f32[_,R]")
def latent_store(x, gain, eps, cache, fb):
    assert x.dtype == cache.dtype
    nv.call("latent_store", nv.ptr(x), I(x.stride(0)), nv.ptr(gain), F(eps), nv.ptr(cache), nv.ptr(fb.out_loc),
            I(x.shape[0]), I(x.shape[1]), _f32(x.dtype))


def latent_tiling(seg_lens, rows: int, heads: int, rank: int, max_context: int, sms: int):
    """(rows per CTA, row tiles, key splits) of the tensor-core kernel.  Splitting the keys pays while the row tiles
    alone leave SMs idle and a tile has several key tiles."""
    lens = seg_lens if seg_lens is not None else [1] * rows
    per_seg = max(lens) * heads
    m = 16 if per_seg <= 16 else 32 if per_seg <= 32 else 64
    tiles = sum(-(-n * heads // m) for n in lens)
    rp = -(-rank // 128) * 128
    smem = m * rp * 2 + 2 * 64 * rp * 2 + m * 68 * 4 + m * 64 * 2 + 16 * m
    ctas = sms * max(1, min(SMEM_BYTES // smem, 4))
    ktiles = -(-max_context // 64)
    return m, tiles, max(1, min(ctas // max(tiles, 1), -(-ktiles // 2), 32))


@tensors(q="bf16|f32[T,H,R]", cache="bf16|f32[_,R]")
def latent_attention(q, cache, fb, scale):
    t, h, r = q.shape
    assert q.dtype == cache.dtype
    o = torch.empty_like(q)
    m = tiles = 0
    nsplit, acc, ml = 1, None, None
    if q.dtype == torch.bfloat16 and r % 8 == 0 and r <= 512:
        m, tiles, nsplit = latent_tiling(fb.seg_lens, t, h, r, fb.max_context, num_sms(q.device))
        if nsplit > 1:
            acc = torch.empty(t * h, nsplit, r, dtype=torch.float32, device=q.device)
            ml = torch.empty(t * h, nsplit, 2, dtype=torch.float32, device=q.device)
    pt = fb.page_table
    nv.call("latent_attention", nv.ptr(q), nv.ptr(cache), nv.ptr(o), nv.ptr(fb.slots), nv.ptr(fb.positions), nv.ptr(pt),
            I(pt.stride(0)), nv.ptr(fb.seg_off), I(0 if fb.seg_off is None else fb.seg_off.shape[0] - 1),
            nv.ptr(fb.num_valid), I(t), I(h), I(r), F(scale), I(m), I(tiles), I(nsplit), nv.ptr(acc), nv.ptr(ml),
            _f32(q.dtype))
    return o


# --------------------------------------------------------------------------- recurrent time mixing
@tensors(x="f32[T,D]", gain="f32[D]", mu="f32[_,D]", prev="f32[S,D]", tail="f32[S,D]")
def shift_mix(x, gain, eps, mu, prev, tail, fb, dtype):
    t, d = x.shape
    n = mu.shape[0]
    out = torch.empty(t, n * d, dtype=dtype, device=x.device)
    nv.call("shift_mix", nv.ptr(x), nv.ptr(gain), F(eps), nv.ptr(mu), I(n), nv.ptr(prev), nv.ptr(tail),
            nv.ptr(fb.slots), nv.ptr(fb.positions), nv.ptr(out), I(t), I(d), _f32(dtype))
    return out


@tensors(p="bf16|f32[T,_]", a="f32[T,N]", w0="f32[N]", u="f32[N]", gain="f32[N]", state="f32[S,_,_,_]",
         prev="f32[S,W]", tail="f32[S,W]")
def wkv(p, a, w0, u, gain, state, prev, tail, fb, heads, eps):
    t, hd = a.shape
    assert p.shape[1] == 4 * hd and state.shape[1] == heads
    out = torch.empty(t, hd, dtype=p.dtype, device=p.device)
    segs = t if fb.seg_off is None else fb.seg_off.shape[0] - 1
    nv.call("wkv_scan", nv.ptr(p), nv.ptr(a), nv.ptr(w0), nv.ptr(u), nv.ptr(gain), nv.ptr(state), nv.ptr(prev),
            nv.ptr(tail), I(prev.shape[1]), nv.ptr(fb.slots), nv.ptr(fb.positions), nv.ptr(fb.seg_off), I(segs),
            I(heads), I(hd // heads), F(eps), nv.ptr(out), _f32(p.dtype))
    return out
