"""Python wrappers around the sm_100a kernels of the layered models (csrc/residual.cu, latent_attn.cu, mingru.cu, wkv.cu,
moe_bf16.cu, gemm_simt.cu), one function per facade op in :mod:`minisgl.ops.api`.  Activations are bf16 or fp32."""
from __future__ import annotations

import os

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
@tensors(ids="i32[T]", weight="bf16[_,D]", feedback="?i32[_]", slots="?i32[T]", table="?bf16[_,D]", positions="?i32[T]",
         pairs="?bf16[_,D]", tokens="?i32[_]")
def embed_residual(ids, weight, dtype, feedback=None, slots=None, want_act=False, mul=1.0, table=None, positions=None,
                   streams=None, pairs=None, pair_mul=(0, 0), tokens=None, fb=None):
    t, d = ids.shape[0], weight.shape[1]
    x = torch.empty(*((t, d) if streams is None else (t, streams, d)), dtype=torch.float32, device=ids.device)
    act = torch.empty(t, d, dtype=dtype, device=ids.device) if want_act else None
    buckets = 1 if pairs is None else pairs.shape[0] - 1
    nv.call("embed_residual", nv.ptr(ids), nv.ptr(feedback), nv.ptr(slots), nv.ptr(weight), nv.ptr(x), nv.ptr(act), F(mul),
            nv.ptr(table), nv.ptr(positions), I(0 if table is None else table.shape[0]), I(streams or 1), nv.ptr(pairs),
            I(buckets), I(pair_mul[0] % buckets), I(pair_mul[1] % buckets), nv.ptr(tokens),
            nv.ptr(None if fb is None else fb.out_loc), nv.ptr(None if fb is None else fb.page_table),
            I(0 if fb is None else fb.page_table.stride(0)), I(t), I(d), _f32(dtype))
    return x, act


@tensors(x="f32[T,S,D]", pre="?f32[_]", post="?f32[_]", sub="?f32[T,D]", rows="?i64[_]")
def stream_norm(x, eps, dtype, pre, post, sub, experts, rows, keep):
    t, s, d = x.shape
    assert (pre is None or pre.shape[0] == s + 1) and (post is None or post.shape[0] == s * (s + 1))
    erows = wts = idx = h = None
    topk = n_experts = 0
    if experts is not None:
        erows, wts, idx, n_experts, h = experts
        topk = idx.shape[1]
        assert erows.dtype == h.dtype == dtype and erows.shape == (t * topk, d) and h.shape == (t, d)
        assert erows.is_contiguous() and h.is_contiguous() and idx.shape == wts.shape == (t, topk)
    n_out = t if rows is None else rows.shape[0]
    out = torch.empty(n_out, d, dtype=dtype, device=x.device) if pre is not None else None
    nv.call("stream_norm", nv.ptr(x), nv.ptr(rows), nv.ptr(post), nv.ptr(sub), nv.ptr(erows), nv.ptr(wts), nv.ptr(idx),
            I(topk), I(n_experts), nv.ptr(h), nv.ptr(pre), F(eps), I(1 if keep and post is not None else 0), nv.ptr(out),
            I(n_out), I(s), I(d), _f32(dtype))
    return out


@tensors(x="f32[_,D]", gain="?f32[D]", rows="?i64[_]", add="?f32[_,D]", add2="?f32[_,D]", vec="?f32[D]")
def residual_norm(x, gain, eps, dtype, mul=1.0, rows=None, add=None, add2=None, vec=None, experts=None, cast=False, sub=None):
    n, d = x.shape
    erows = wts = idx = None
    topk = 0
    if experts is not None:
        erows, wts, idx = experts
        topk = idx.shape[1]
        assert erows.dtype == dtype and erows.shape == (n * topk, d) and erows.is_contiguous()
    y = bias = sub_gain = None
    if sub is not None:
        y, bias, sub_gain = sub
        assert y.shape == (n, d) and y.dtype == torch.float32 and y.is_contiguous()
        assert all(v is None or (v.shape == (d,) and v.dtype == torch.float32) for v in (bias, sub_gain))
    n_out = n if rows is None else rows.shape[0]
    out = torch.empty(n_out, d, dtype=dtype, device=x.device) if gain is not None or cast else None
    nv.call("residual_norm", nv.ptr(x), nv.ptr(rows), nv.ptr(y), nv.ptr(bias), nv.ptr(sub_gain), nv.ptr(add), nv.ptr(add2), nv.ptr(vec), nv.ptr(erows),
            nv.ptr(wts), nv.ptr(idx), I(topk), nv.ptr(gain), F(eps), F(mul), nv.ptr(out), I(n_out), I(d), _f32(dtype))
    return out


# --------------------------------------------------------------------------- mixture of experts
ROUTERS = {"selected": 3, "softmax": 4}      # csrc/moe.cu: moe_topk_kernel


@tensors(h="bf16|f32[T,D]", weight="bf16[E,D]", bias="f32[E]", num_valid="?i32[1]")
def route_topk(h, weight, bias, top, num_valid=None, kind="selected", scale=1.0):
    t, e = h.shape[0], weight.shape[0]
    if _tma_ok(h, weight, h.shape[1]):
        scores = gemm_bf16_partials(h, weight)      # [S, T, E]; the selection kernel adds the splits
    else:
        scores = linear(h, weight, out_dtype=torch.float32)[None]
    idx = torch.empty(t, top, dtype=torch.int32, device=h.device)
    wts = torch.empty(t, top, dtype=torch.float32, device=h.device)
    nv.call("moe_topk", nv.ptr(scores), nv.ptr(bias), nv.ptr(None), nv.ptr(None), nv.ptr(num_valid), nv.ptr(idx),
            nv.ptr(wts), I(t), I(e), I(top), F(scale), I(ROUTERS[kind]), I(scores.shape[0]), L(scores.stride(0)))
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
        xs, sms = new(d), I(num_sms(h.device))
        nv.call("moe_gather_rows", nv.ptr(h), nv.ptr(xs), nv.ptr(plan), I(routes), I(max_tiles), I(top), I(d))
        nv.call("moe_bf16_gemm", I(1), I(nt), nv.ptr(w13), nv.ptr(xs), nv.ptr(plan), I(routes), I(max_tiles),
                nv.ptr(act), I(e), I(f), I(d), sms)
        nv.call("moe_bf16_gemm", I(2), I(nt), nv.ptr(w2), nv.ptr(act), nv.ptr(plan), I(routes), I(max_tiles),
                nv.ptr(rows), I(e), I(d), I(f), sms)
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


@tensors(p="bf16|f32[T,_]s", gain="f32[R]", freq="f32[_]", cache="bf16|f32[_,_]")
def latent_rotate_store(p, at_rot, at_c, gain, eps, freq, mul, cache, fb, heads, dim, whole):
    t, rank, rot = p.shape[0], gain.shape[0], 2 * freq.shape[0]
    assert p.dtype == cache.dtype and cache.shape[1] == rank + rot and p.shape[1] >= at_c + rank + rot
    q = torch.empty(t, heads * (dim + rot), dtype=p.dtype, device=p.device) if whole else None
    nv.call("latent_rotate_store", nv.ptr(p), I(p.stride(0)), I(at_rot), I(at_c), nv.ptr(gain), F(eps), nv.ptr(freq), F(mul),
            nv.ptr(fb.positions), nv.ptr(fb.out_loc), nv.ptr(cache), nv.ptr(q), I(t), I(heads), I(dim), I(rot), I(rank),
            _f32(p.dtype))
    return q


def latent_tiling(seg_lens, rows: int, heads: int, rank: int, max_context: int, sms: int):
    """(rows per CTA, row tiles, key splits) of the tensor-core kernel.  rank: values of a cache row.  Splitting the keys pays while the row tiles
    alone leave SMs idle and a tile has several key tiles."""
    lens = seg_lens if seg_lens is not None else [1] * rows
    per_seg = max(lens) * heads
    m = 16 if per_seg <= 16 else 32 if per_seg <= 32 or rank > 512 else 64
    tiles = sum(-(-n * heads // m) for n in lens)
    rp = -(-rank // 128) * 128
    smem = m * rp * 2 + 2 * 64 * rp * 2 + m * 68 * 4 + m * 64 * 2 + 20 * m
    ctas = sms * max(1, min(SMEM_BYTES // smem, 4))
    ktiles = -(-max_context // 64)
    return m, tiles, max(1, min(ctas // max(tiles, 1), -(-ktiles // 2), 32))


@tensors(q="bf16|f32[T,H,R]", cache="bf16|f32[_,_]", q_rot="?bf16|f32[T,_]s")
def latent_attention(q, cache, fb, scale, q_rot, window):
    t, h, r = q.shape
    width = cache.shape[1]
    assert q.dtype == cache.dtype and width - r == (0 if q_rot is None else q_rot.shape[1] // h)
    o = torch.empty_like(q)
    m = tiles = 0
    nsplit, acc, ml = 1, None, None
    even = r % 8 == 0 and width % 8 == 0 and width <= 640 and (q_rot is None or (q_rot.stride(0) % 8 == 0 and q_rot.data_ptr() % 16 == 0))
    if q.dtype == torch.bfloat16 and even:
        m, tiles, nsplit = latent_tiling(fb.seg_lens, t, h, width, window_span(fb, window), num_sms(q.device))
        if nsplit > 1:
            acc = torch.empty(t * h, nsplit, r, dtype=torch.float32, device=q.device)
            ml = torch.empty(t * h, nsplit, 2, dtype=torch.float32, device=q.device)
    pt = fb.page_table
    nv.call("latent_attention", nv.ptr(q), nv.ptr(cache), nv.ptr(o), nv.ptr(fb.slots), nv.ptr(fb.positions), nv.ptr(pt),
            I(pt.stride(0)), nv.ptr(fb.seg_off), I(0 if fb.seg_off is None else fb.seg_off.shape[0] - 1),
            nv.ptr(fb.num_valid), I(t), I(h), I(r), nv.ptr(q_rot), I(0 if q_rot is None else q_rot.stride(0)), I(width - r),
            I(window), F(scale), I(m), I(tiles), I(nsplit), nv.ptr(acc), nv.ptr(ml), _f32(q.dtype))
    return o


# MINISGL_LATENT_PREFILL: auto (by cost), expanded (wherever the kernel can) or absorbed
LATENT_PREFILL = os.environ.get("MINISGL_LATENT_PREFILL", "auto")
EXPAND_BYTES = 4 << 30                        # bound of the expanded keys and values of one call
ABSORBED_TFLOPS, EXPANDED_TFLOPS, GEMM_TFLOPS, EXPAND_US = 200.0, 900.0, 600.0, 25.0    # measured rates


def window_span(fb, window: int, tile_tokens: int = 1) -> int:
    """The most keys that a tile of so many tokens reads."""
    return min(fb.max_context, window + tile_tokens - 1) if window else fb.max_context


def prefers_expanded(q_dtype, fb, heads: int, dim: int, vdim: int, rank: int, rot: int = 0, window: int = 0) -> bool:
    """Whether a prefill forward should expand its requests' latents to keys and values (csrc/flash_attn.cu) instead of
    attending over the latents: expanding costs every request's whole context once, and then a query pays dim + vdim per
    key instead of twice the rank."""
    if fb.seg_ends is None or q_dtype != torch.bfloat16 or LATENT_PREFILL == "absorbed":
        return False
    wide = dim + rot                 # of a query and an expanded key
    if wide % 8 or vdim % 8 or rank % 8 or rot % 8 or wide > 128 or vdim > 128:
        return False
    reach = window or max(fb.seg_ends)
    need = [min(s, n + reach - 1) for n, s in zip(fb.seg_lens, fb.seg_ends)]         # keys that a portion sees
    ctx = sum(-(-s // KV_ALIGN) * KV_ALIGN for s in need)
    if 2 * ctx * (heads * (wide + vdim) + rank + rot) > EXPAND_BYTES:
        return False
    if LATENT_PREFILL == "expanded":
        return True
    each = [min(s - n / 2, reach) for n, s in zip(fb.seg_lens, fb.seg_ends)]         # keys that a query sees, on average
    pairs = sum(n * k for n, k in zip(fb.seg_lens, each))
    tiled = sum(-(-n // 256) * 256 * (k + (192 if window else 64)) for n, k in zip(fb.seg_lens, each))
    absorbed = 2e-6 * heads * (2 * rank + rot) * pairs / ABSORBED_TFLOPS \
        + 2e-6 * sum(fb.seg_lens) * heads * rank * (dim + vdim) / GEMM_TFLOPS
    expanded = 2e-6 * heads * ((wide + vdim) * tiled / EXPANDED_TFLOPS
                               + ctx * (wide * (rank + rot) + vdim * rank) / GEMM_TFLOPS) + EXPAND_US
    return expanded < absorbed


KV_ALIGN = 64       # a request's expanded keys start at a multiple of this (16-byte TMA boundaries of V^T)


def prompt_items(row: int, n: int, s: int, at: int, window: int = 0):
    """Work items of the prompt kernel for a portion of ``n`` queries from row ``row`` on, the last ones of ``s`` keys that stand from
    row ``at`` on: (first query row, queries, place of the first among the item's keys, first key row, keys).  With a window an item's
    keys begin where its first query's do, rounded down so that TMA can fetch them."""
    for q in range(0, n, 256):
        m, pos = min(256, n - q), s - n + q
        skip = max(0, pos - window + 1) // KV_ALIGN * KV_ALIGN if window else 0
        yield row + q, m, pos - skip, at + skip, pos - skip + m


def _expanded_plan(fb, device, window: int):
    """(request list [n, 4], work items [m, 5], expanded rows), one per forward: the same for all layers of a window.  Items are
    ordered by the number of keys they see, longest first."""
    plans = fb.__dict__.setdefault("expanded_plans", {})
    plan = plans.get(window)
    if plan is None:
        reqs, items, at, row = [], [], 0, 0
        for n, s, slot in zip(fb.seg_lens, fb.seg_ends, fb.seg_slots):
            key0 = max(0, s - n - window + 1) if window else 0
            reqs.append((slot, s - key0, at, key0))
            items += prompt_items(row, n, s - key0, at, window)
            at += -(-(s - key0) // KV_ALIGN) * KV_ALIGN
            row += n
        items.sort(key=lambda i: -i[4])
        host = torch.tensor([v for t in (*reqs, *items) for v in t], dtype=torch.int32).pin_memory()
        dev = host.to(device, non_blocking=True)
        k = 4 * len(reqs)
        plan = plans[window] = (dev[:k], dev[k:], len(reqs), len(items), at)
    return plan


@tensors(q="bf16[_,_]s", cache="bf16[_,W]", uk="bf16[_,W]", uv="bf16[_,_]")
def expanded_attention(q, cache, fb, uk, uv, heads, scale, window):
    t, dim, vdim, width, rank = q.shape[0], uk.shape[0] // heads, uv.shape[0] // heads, cache.shape[1], uv.shape[1]
    reqs, items, n_reqs, n_items, rows = _expanded_plan(fb, q.device, window)
    ctx = torch.empty(rows, width, dtype=q.dtype, device=q.device)
    pt = fb.page_table
    nv.call("latent_gather", nv.ptr(cache), nv.ptr(ctx), nv.ptr(reqs), I(n_reqs), I(rows), nv.ptr(pt), I(pt.stride(0)),
            I(width))
    k, vt = linear(ctx, uk), linear(uv, ctx[:, :rank])
    out = torch.empty(t, heads * vdim, dtype=q.dtype, device=q.device)
    nv.call("flash_attention", nv.ptr(q), I(q.stride(0)), nv.ptr(k), nv.ptr(vt), nv.ptr(out), nv.ptr(items), I(n_items),
            I(t), I(rows), I(heads), I(heads), I(dim), I(vdim), F(scale), F(0.0), nv.ptr(None), nv.ptr(None), I(0), nv.ptr(None), nv.ptr(None),
            I(window), nv.ptr(None), nv.ptr(None), I(0))
    return out


# --------------------------------------------------------------------------- element-wise recurrence
GRU_TILES = (32, 16, 8)          # elements per CTA of the parallel form


@tensors(p="f32[T,_]s", bias_z="f32[W]", bias_u="f32[W]", state="f32[_,W]")
def mingru(p, at_u, at_g, bias_z, bias_u, state, fb, dtype):
    t, width = p.shape[0], state.shape[1]
    assert p.shape[1] >= at_g + width
    y = torch.empty(t, width, dtype=dtype, device=p.device)
    segs = t if fb.seg_off is None else fb.seg_off.shape[0] - 1
    fill = num_sms(p.device) * 4 // 3
    ct = next((c for c in GRU_TILES if -(-width // c) * segs >= fill), GRU_TILES[-1])
    nv.call("mingru", nv.ptr(p), I(p.stride(0)), I(at_u), I(at_g), nv.ptr(bias_z), nv.ptr(bias_u), nv.ptr(state), nv.ptr(y),
            nv.ptr(fb.slots), nv.ptr(fb.positions), nv.ptr(fb.seg_off), I(segs),
            nv.ptr(fb.num_valid if fb.seg_off is None else None), I(max(fb.seg_lens) if fb.seg_lens is not None else 1), I(ct),
            I(width), _f32(dtype))
    return y


# --------------------------------------------------------------------------- recurrent time mixing
@tensors(x="f32[T,D]", gain="f32[D]", mu="f32[_,D]", prev="f32[S,D]", tail="f32[S,D]")
def shift_mix(x, gain, eps, mu, prev, tail, fb, dtype):
    t, d = x.shape
    n = mu.shape[0]
    out = torch.empty(t, n * d, dtype=dtype, device=x.device)
    nv.call("shift_mix", nv.ptr(x), nv.ptr(gain), F(eps), nv.ptr(mu), I(n), nv.ptr(prev), nv.ptr(tail),
            nv.ptr(fb.slots), nv.ptr(fb.positions), nv.ptr(out), I(t), I(d), _f32(dtype))
    return out


# Portions of at least WKV_CHUNK_MIN tokens run the recurrence in chunks (csrc/wkv_chunk.cu).  In 32-bit serving it stays
# token by token: decays are then products of the decays themselves, not exponentials of sums.  WKV_CHUNKED overrides.
WKV_CHUNKED = None
WKV_CHUNK_MIN, WKV_CHUNK = 64, 32


def _chunk_plan(fb, device, size=WKV_CHUNK):
    """(chunks [n, 2], segments [m, 4]) of a forward for a recurrence in chunks of ``size``; the same for all layers."""
    plans = fb.__dict__.setdefault("chunk_plans", {})
    plan = plans.get(size)
    if plan is None:
        chunks, segs, row = [], [], 0
        for n, slot in zip(fb.seg_lens, fb.seg_slots):
            c0 = len(chunks)
            chunks += [(row + i, min(size, n - i)) for i in range(0, n, size)]
            segs.append((slot, c0, len(chunks) - c0, row))
            row += n
        host = torch.tensor([v for t in (*chunks, *segs) for v in t], dtype=torch.int32).pin_memory()
        dev = host.to(device, non_blocking=True)
        k = 2 * len(chunks)
        plan = plans[size] = (dev[:k], dev[k:], len(chunks), len(segs))
    return plan


@tensors(p="bf16|f32[T,_]", a="f32[T,N]", w0="f32[N]", u="f32[N]", gain="f32[N]", state="f32[S,_,_,_]",
         prev="f32[S,W]", tail="f32[S,W]")
def wkv(p, a, w0, u, gain, state, prev, tail, fb, heads, eps):
    t, hd = a.shape
    assert p.shape[1] == 4 * hd and state.shape[1] == heads
    out = torch.empty(t, hd, dtype=p.dtype, device=p.device)
    chunked = WKV_CHUNKED if WKV_CHUNKED is not None else p.dtype == torch.bfloat16
    if chunked and fb.seg_lens is not None and max(fb.seg_lens) >= WKV_CHUNK_MIN:
        d = hd // heads
        chunks, segs, n_chunks, n_segs = _chunk_plan(fb, p.device)
        us = torch.empty(n_chunks, heads, d, d, dtype=torch.float32, device=p.device)
        decay = torch.empty(n_chunks, heads, d, dtype=torch.float32, device=p.device)
        nv.call("wkv_chunked", nv.ptr(p), nv.ptr(a), nv.ptr(w0), nv.ptr(u), nv.ptr(gain), nv.ptr(state), nv.ptr(prev),
                nv.ptr(tail), I(prev.shape[1]), nv.ptr(fb.positions), nv.ptr(fb.seg_off), nv.ptr(chunks), I(n_chunks),
                nv.ptr(segs), I(n_segs), nv.ptr(us), nv.ptr(decay), I(heads), I(d), F(eps), nv.ptr(out), _f32(p.dtype))
        return out
    segs = t if fb.seg_off is None else fb.seg_off.shape[0] - 1
    nv.call("wkv_scan", nv.ptr(p), nv.ptr(a), nv.ptr(w0), nv.ptr(u), nv.ptr(gain), nv.ptr(state), nv.ptr(prev),
            nv.ptr(tail), I(prev.shape[1]), nv.ptr(fb.slots), nv.ptr(fb.positions), nv.ptr(fb.seg_off), I(segs),
            I(heads), I(hd // heads), F(eps), nv.ptr(out), _f32(p.dtype))
    return out
