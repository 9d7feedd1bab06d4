"""The kernels of the layered models, one mechanism at a time, against the plain statements in ``plain_bedalorn``."""
import math

import pytest
import torch

import plain_bedalorn as P
from layered_util import make_fb
from minisgl.ops import api as O
from minisgl.ops import cuda_layers as C

pytestmark = pytest.mark.gpu
DEV = "cuda"
F = torch.float64
TOL = {torch.bfloat16: 1.2e-2, torch.float32: 2e-5}
BOTH = pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])


def rand(*shape, seed=0, std=1.0, dtype=torch.float32):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * std).to(dtype)


def err(got, want):
    return P.rel_err(got, want)


# --------------------------------------------------------------------------- residual stream
@BOTH
@pytest.mark.parametrize("d", [96, 100, 4096, 9000, 33])
def test_residual_norm(d, dtype):
    n, top = 7, 3
    x, gain, add, vec = rand(n, d), rand(d, seed=1), rand(n, d, seed=2), rand(d, seed=3)
    rows, wts = rand(n * top, d, seed=4).to(dtype), rand(n, top, seed=5)
    idx = torch.randint(0, 5, (n, top), dtype=torch.int32)
    idx[2, 1] = -1
    want = x.to(F) + add.to(F) + 2 * vec.to(F) * 0.5
    w = torch.where(idx < 0, torch.zeros_like(wts), wts).to(F)
    want = want + (rows.to(F).view(n, top, d) * w[..., None]).sum(1)
    xc = x.to(DEV)
    h = O.residual_norm(xc, gain.to(DEV), 1e-3, dtype, mul=1.7, add=add.to(DEV), vec=vec.to(DEV),
                        experts=(rows.to(DEV), wts.to(DEV), idx.to(DEV)))
    assert err(xc, want) < 1e-6
    assert err(h, P.rms(want, 1e-3) * gain.to(F) * 1.7) < TOL[dtype]
    pick = torch.tensor([5, 0, 5])
    assert err(O.residual_norm(xc, gain.to(DEV), 1e-3, dtype, rows=pick.to(DEV)),
               (P.rms(want, 1e-3) * gain.to(F))[pick]) < TOL[dtype]
    before = xc.clone()
    assert O.residual_norm(xc, None, 1e-3, dtype, vec=vec.to(DEV)) is None
    assert torch.allclose(xc, before + vec.to(DEV))
    assert torch.equal(O.residual_norm(xc, None, 1e-3, dtype, cast=True), xc.to(dtype))


@BOTH
@pytest.mark.parametrize("m,k,n,act", [(5, 96, 40, "relu2"), (130, 72, 33, None), (64, 12, 100, "tanh"),
                                       (300, 264, 520, None), (1, 20, 7, "relu2")])
def test_linear(m, k, n, act, dtype):
    """Row lengths TMA can and cannot fetch, activations in the epilogue, accumulation into fp32."""
    x, w = rand(m, k).to(dtype), rand(n, k, seed=1, std=k ** -0.5, dtype=torch.bfloat16)
    y = x.to(F) @ w.to(F).T
    y = {"relu2": lambda v: v.clamp_min(0) ** 2, "tanh": torch.tanh, None: lambda v: v}[act](y)
    out = O.linear(x.to(DEV), w.to(DEV), out_dtype=torch.float32, act=act)
    assert err(out, y) < 2e-5
    base = rand(m, n, seed=2)
    acc = base.to(DEV)
    O.linear(x.to(DEV), w.to(DEV), out=acc, accumulate=True, act=act)
    assert err(acc, y + base.to(F)) < 2e-5


@pytest.mark.parametrize("m,k,n,groups,act", [(4000, 72, 1030, 1, "relu2"), (1300, 200, 2600, 1, None), (2050, 40, 264, 7, "tanh"),
                                              (129, 64, 13000, 1, None)])
def test_projections_of_many_rows(m, k, n, groups, act):
    """The persistent kernel: ragged tiles in every direction, batches, fp32 accumulation and bf16 results."""
    from minisgl.ops.gemm import PREFILL_MIN_TILES, prefill_tiles

    assert prefill_tiles(m, n, groups) >= PREFILL_MIN_TILES
    x, w = rand(m, groups * k + 8, dtype=torch.bfloat16), rand(groups * n, k, seed=1, std=k ** -0.5, dtype=torch.bfloat16)
    f = {"relu2": lambda v: v.clamp_min(0) ** 2, "tanh": torch.tanh, None: lambda v: v}[act]
    want = f(torch.cat([x[:, i * k:(i + 1) * k].float() @ w[i * n:(i + 1) * n].float().T for i in range(groups)], 1))
    xs = x.to(DEV)[:, : groups * k]
    assert err(O.grouped_linear(xs, w.to(DEV), groups, act=act), want) < 1e-2
    base = rand(m, groups * n, seed=2)
    acc = base.to(DEV)
    O.grouped_linear(xs, w.to(DEV), groups, out=acc, accumulate=True, act=act)
    assert err(acc, want + base) < 1e-4


@BOTH
def test_grouped_linear_reads_column_slices(dtype):
    t, groups, k, n = 70, 3, 40, 24
    wide, w = rand(t, groups * k + 64).to(dtype), rand(groups * n, k, seed=1, dtype=torch.bfloat16)
    got = O.grouped_linear(wide.to(DEV)[:, : groups * k], w.to(DEV), groups)
    for i in range(groups):
        want = wide[:, i * k:(i + 1) * k].to(F) @ w[i * n:(i + 1) * n].to(F).T
        assert err(got[:, i * n:(i + 1) * n], want) < TOL[dtype]


# --------------------------------------------------------------------------- latent attention
def attention_case(heads, rank, segs, dtype, prefill=True, seed=0, ps=16):
    fb, rows = make_fb(segs, DEV, ps=ps, seed=seed, prefill=prefill)
    t = fb.positions.shape[0]
    q, cache = rand(t, heads, rank, seed=seed).to(dtype), rand(rows, rank, seed=seed + 1).to(dtype)
    return fb, q, cache


def plain_attention(q, cache, fb, scale):
    table, slots, pos = fb.page_table.cpu().long(), fb.slots.cpu().long(), fb.positions.cpu()
    out = torch.empty(q.shape, dtype=F)
    for i in range(q.shape[0]):
        c = cache[table[slots[i], : int(pos[i]) + 1]].to(F)
        out[i] = torch.softmax(q[i].to(F) @ c.T * scale, -1) @ c
    return out


SEGS = [[(0, 0, 1)], [(1, 0, 70)], [(2, 63, 2), (0, 0, 5), (3, 200, 130)], [(4, 1000, 3), (1, 0, 200), (2, 15, 1)]]


@BOTH
@pytest.mark.parametrize("heads,rank", [(1, 8), (3, 48), (5, 136), (16, 128), (20, 264), (40, 512), (70, 40), (2, 20)])
@pytest.mark.parametrize("segs", SEGS)
def test_latent_attention_prefill(heads, rank, segs, dtype):
    fb, q, cache = attention_case(heads, rank, segs, dtype)
    scale = 0.7 / math.sqrt(rank)
    got = O.latent_attention(q.to(DEV), cache.to(DEV), fb, scale)
    assert err(got.flatten(0, 1), plain_attention(q, cache, fb, scale).flatten(0, 1)) < TOL[dtype]


@BOTH
@pytest.mark.parametrize("heads,rank", [(4, 96), (24, 128), (6, 520), (128, 256)])
def test_latent_attention_decode(heads, rank, dtype):
    """Single rows at, before and behind page and key-tile borders; with and without split keys."""
    segs = [(0, 0, 1), (1, 15, 1), (2, 16, 1), (3, 63, 1), (4, 64, 1), (5, 1700, 1)]
    fb, q, cache = attention_case(heads, rank, segs, dtype, prefill=False)
    want = plain_attention(q, cache, fb, 0.05)
    got = O.latent_attention(q.to(DEV), cache.to(DEV), fb, 0.05)
    assert err(got.flatten(0, 1), want.flatten(0, 1)) < TOL[dtype]
    fb.max_context = 1        # one split
    assert err(O.latent_attention(q.to(DEV), cache.to(DEV), fb, 0.05).flatten(0, 1), want.flatten(0, 1)) < TOL[dtype]


@BOTH
@pytest.mark.parametrize("far", [0, 1, 15, 16, 63, 64, 700])
def test_one_key_stands_out(far, dtype):
    """A query that is almost a multiple of one far key: a key that is missed, or taken from a wrong page, shows."""
    n, heads, rank = 701, 2, 64
    for prefill in (False, True):
        fb, rows = make_fb([(2, n - 1, 1)] if not prefill else [(2, n - 9, 9)], DEV, prefill=prefill)
        t = fb.positions.shape[0]
        cache = rand(rows, rank, seed=3).to(dtype)
        loc = int(fb.page_table[2, far])
        q = (cache[loc].float() * 8).to(dtype).expand(t, heads, rank).contiguous()
        got = O.latent_attention(q.to(DEV), cache.to(DEV), fb, 1.0)
        want = plain_attention(q, cache, fb, 1.0)
        assert err(got.flatten(0, 1), want.flatten(0, 1)) < TOL[dtype]
        if far <= n - 9:
            assert err(want[-1, :1], cache[loc].to(F)[None]) < 1e-3


def test_padded_rows_are_left_alone():
    fb, q, cache = attention_case(3, 64, [(0, 5, 1), (1, 9, 1), (6, 0, 1), (6, 0, 1)], torch.bfloat16, prefill=False)
    fb.num_valid = torch.tensor([2], dtype=torch.int32, device=DEV)
    got = O.latent_attention(q.to(DEV), cache.to(DEV), fb, 0.1)
    assert err(got[:2].flatten(0, 1), plain_attention(q, cache, fb, 0.1)[:2].flatten(0, 1)) < 1.2e-2


@pytest.mark.parametrize("heads,dim,vdim,rank", [(1, 8, 8, 16), (3, 24, 40, 48), (2, 64, 80, 136), (4, 128, 128, 512),
                                                 (5, 72, 120, 64)])
@pytest.mark.parametrize("segs", SEGS + [[(0, 0, 600)], [(1, 127, 129), (2, 128, 257), (3, 1, 255), (4, 500, 256)]])
def test_expanded_attention(heads, dim, vdim, rank, segs):
    """Keys and values expanded from the latents: same attention, tcgen05."""
    fb, rows = make_fb(segs, DEV)
    t = fb.positions.shape[0]
    bf = torch.bfloat16
    cache = rand(rows, rank, seed=1, dtype=bf)
    uk, uv = rand(heads * dim, rank, seed=2, std=rank ** -0.5, dtype=bf), rand(heads * vdim, rank, seed=3, std=rank ** -0.5, dtype=bf)
    wide = rand(t, heads * dim + rank, seed=4, dtype=bf)
    scale = 1.5 / math.sqrt(dim)
    got = O.expanded_attention(wide.to(DEV)[:, : heads * dim], cache.to(DEV), fb, uk.to(DEV), uv.to(DEV), heads, scale)
    q = wide[:, : heads * dim].to(F).view(t, heads, dim)
    table, slots, pos = fb.page_table.cpu().long(), fb.slots.cpu().long(), fb.positions.cpu()
    worst = 0.0
    for i in list(range(0, t, 37)) + [t - 1]:
        c = cache[table[slots[i], : int(pos[i]) + 1]].to(F)
        k, v = (c @ uk.to(F).T).view(-1, heads, dim), (c @ uv.to(F).T).view(-1, heads, vdim)
        p = torch.softmax(torch.einsum("hd,jhd->hj", q[i], k) * scale, -1)
        worst = max(worst, err(got[i].view(heads, vdim), torch.einsum("hj,jhv->hv", p, v)))
    assert worst < 2e-2


@pytest.mark.parametrize("far", [0, 63, 127, 128, 300])
def test_expanded_attention_far_key_and_growing_maximum(far):
    """One key far back dominates late queries, so the running maximum has to be right whichever tile it sits in."""
    heads, dim, rank, n = 2, 64, 64, 520
    fb, rows = make_fb([(3, 0, n)], DEV)
    bf = torch.bfloat16
    cache = rand(rows, rank, seed=1, dtype=bf)
    eye = torch.eye(rank).repeat(heads, 1).to(bf)
    key = cache[int(fb.page_table[3, far])]
    q = (key.float() * 4).to(bf).repeat(n, heads)
    got = O.expanded_attention(q.to(DEV), cache.to(DEV), fb, eye.to(DEV), eye.to(DEV), heads, 1.0)
    want = plain_attention(q.view(n, heads, dim), cache, fb, 1.0)
    assert err(got.view(n * heads, dim), want.flatten(0, 1)) < 2e-2
    assert err(want[-1, :1], key.to(F)[None]) < 1e-3


@BOTH
def test_latent_store(dtype):
    fb, rows = make_fb([(1, 14, 5), (2, 0, 3)], DEV)
    rank = 52
    fb.out_loc[3] = -1
    x, gain = rand(8, rank + 12).to(dtype), rand(rank, seed=1)
    cache = torch.full((rows, rank), 7.0, dtype=dtype, device=DEV)
    O.latent_store(x.to(DEV)[:, 12:], gain.to(DEV), 1e-2, cache, fb)
    want = torch.full((rows, rank), 7.0, dtype=F)
    for i in range(8):
        if i != 3:
            want[int(fb.out_loc[i])] = P.rms(x[i, 12:].to(F), 1e-2) * gain.to(F)
    assert err(cache, want) < TOL[dtype]


# --------------------------------------------------------------------------- recurrent time mixing
def plain_shift_mix(x, gain, eps, mu, prev):
    h = P.rms(x.to(F), eps) * gain.to(F)
    hp = P.token_shift(h, prev.to(F))
    return torch.cat([h + (hp - h) * m.to(F) for m in mu], -1), h[-1]


@BOTH
@pytest.mark.parametrize("d", [96, 50, 1024])
def test_shift_mix(d, dtype):
    """First rows of a request, of a later portion and single rows; what every portion leaves in its slot."""
    segs = [(0, 0, 3), (1, 7, 4), (2, 0, 1), (3, 9, 1)]
    fb, _ = make_fb(segs, DEV)
    x, gain, mu = rand(9, d), rand(d, seed=1), rand(5, d, seed=2)
    prev, tail = rand(7, d, seed=3), torch.full((7, d), 9.0)
    pc, tc = prev.to(DEV), tail.to(DEV)
    got = O.shift_mix(x.to(DEV), gain.to(DEV), 1e-3, mu.to(DEV), pc, tc, fb, dtype)
    row = 0
    for slot, start, n in segs:
        want, last = plain_shift_mix(x[row:row + n], gain, 1e-3, mu, prev[slot] if start else torch.zeros(d))
        assert err(got[row:row + n], want) < TOL[dtype]
        assert err((pc if n == 1 else tc)[slot][None], last[None]) < 1e-5
        row += n


def wkv_case(segs, heads, d, dtype, seed=0, w0=None):
    fb, _ = make_fb(segs, DEV)
    t, hd = sum(n for _, _, n in segs), heads * d
    p, a = rand(t, 4 * hd, seed=seed).to(dtype), rand(t, hd, seed=seed + 1)
    w0 = rand(hd, seed=seed + 2) - 2.0 if w0 is None else torch.full((hd,), float(w0))
    u, gain = rand(hd, seed=seed + 3), rand(hd, seed=seed + 4)
    state, prev, tail = rand(7, heads, d, d, seed=seed + 5), rand(7, 64, seed=seed + 6), rand(7, 64, seed=seed + 7)
    return fb, p, a, w0, u, gain, state, prev, tail


def check_wkv(segs, heads, d, dtype, tol, w0=None):
    fb, p, a, w0, u, gain, state, prev, tail = wkv_case(segs, heads, d, dtype, w0=w0)
    hd = heads * d
    sc, pc = state.to(DEV), prev.to(DEV)
    got = O.wkv(p.to(DEV), a.to(DEV), w0.to(DEV), u.to(DEV), gain.to(DEV), sc, pc, tail.to(DEV), fb, heads, 1e-4)
    row = 0
    for slot, start, n in segs:
        r, k, v, g = (c.reshape(n, heads, d) for c in p[row:row + n].to(F).split(hd, 1))
        w = torch.exp(-torch.exp(a[row:row + n].to(F) + w0.to(F))).view(n, heads, d)
        s0 = state[slot].to(F) if start else torch.zeros(heads, d, d, dtype=F)
        o, s = P.wkv_recurrence(r, k, v, w, u.to(F).view(heads, d), s0)
        want = (P.rms(o, 1e-4) * gain.to(F).view(heads, d) * P.silu(g)).reshape(n, hd)
        assert err(got[row:row + n], want) < tol
        assert err(sc[slot].flatten(0, 1), s.flatten(0, 1)) < 3e-5
        assert torch.equal(pc[slot].cpu(), tail[slot] if n > 1 else prev[slot])
        row += n


WKV_SEGS = [[(0, 0, 1), (1, 5, 1)], [(2, 0, 40)], [(3, 8, 17), (0, 0, 2), (5, 1, 1), (4, 100, 33)]]


@BOTH
@pytest.mark.parametrize("heads,d", [(1, 8), (3, 16), (2, 20), (2, 32), (2, 41), (2, 64), (1, 128)])
@pytest.mark.parametrize("segs", WKV_SEGS)
def test_wkv_token_by_token(heads, d, segs, dtype):
    check_wkv(segs, heads, d, dtype, TOL[dtype])


@BOTH
@pytest.mark.parametrize("heads,d", [(1, 8), (3, 16), (2, 20), (2, 32), (2, 41), (2, 64), (1, 128)])
@pytest.mark.parametrize("segs", [[(1, 0, 64)], [(2, 3, 200)], [(3, 8, 65), (0, 0, 2), (5, 1, 1), (4, 100, 33), (1, 0, 96)]])
def test_wkv_in_chunks(heads, d, segs, dtype, monkeypatch):
    monkeypatch.setattr(C, "WKV_CHUNKED", True)
    check_wkv(segs, heads, d, dtype, TOL[dtype])


@pytest.mark.parametrize("w0", [-12, -1, 2, 6])
def test_wkv_chunks_with_slow_and_fast_decays(w0, monkeypatch):
    """A state that hardly decays over hundreds of tokens, and decays that leave nothing of the token before."""
    monkeypatch.setattr(C, "WKV_CHUNKED", True)
    check_wkv([(1, 0, 300), (2, 50, 70)], 2, 32, torch.float32, 1e-4, w0=w0)


# --------------------------------------------------------------------------- mixture of experts
@BOTH
@pytest.mark.parametrize("experts,top", [(1, 1), (5, 2), (8, 8), (40, 1), (100, 6)])
def test_router(experts, top, dtype):
    t, d = 33, 72
    h, w, b = rand(t, d).to(dtype), rand(experts, d, seed=1, dtype=torch.bfloat16), rand(experts, seed=2)
    idx, wts = O.route_topk(h.to(DEV), w.to(DEV), b.to(DEV), top)
    z = h.to(F) @ w.to(F).T + b.to(F)
    want = torch.sort(z, -1, descending=True).indices[:, :top]
    assert torch.equal(idx.cpu().long(), want)
    assert err(wts, torch.softmax(torch.gather(z, 1, want), -1)) < 1e-5


def test_router_bias_changes_the_choice_and_the_weights():
    h = torch.zeros(1, 16, dtype=torch.bfloat16, device=DEV)
    w = torch.zeros(4, 16, dtype=torch.bfloat16, device=DEV)
    idx, wts = O.route_topk(h, w, torch.tensor([0.0, 3.0, -1.0, 2.0], device=DEV), 2)
    assert idx.tolist() == [[1, 3]]
    assert torch.allclose(wts.cpu(), torch.softmax(torch.tensor([[3.0, 2.0]]), -1), atol=1e-6)


@BOTH
@pytest.mark.parametrize("t,d,f,experts,top", [(1, 64, 40, 3, 2), (9, 96, 72, 5, 2), (60, 136, 200, 4, 3), (300, 64, 48, 4, 2),
                                               (700, 256, 136, 6, 4), (20, 50, 36, 3, 1)])
def test_experts(t, d, f, experts, top, dtype):
    """Every route-tile width, sizes that fill no tile, experts without a token, rows whose ids are -1."""
    h = rand(t, d).to(dtype)
    w13 = rand(experts, 2, f, d, seed=1, std=d ** -0.5, dtype=torch.bfloat16)
    w2 = rand(experts, d, f, seed=2, std=f ** -0.5, dtype=torch.bfloat16)
    g = torch.Generator().manual_seed(5)
    idx = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(t)]).to(torch.int32)
    idx[idx == 1] = 0 if top == 1 else idx[idx == 1]
    if t > 4:
        idx[3] = -1
    wts = rand(t, top, seed=6)
    got = O.gated_experts(h.to(DEV), idx.to(DEV), wts.to(DEV), w13.to(DEV), w2.to(DEV)).view(t, top, d)
    for i in range(0, t, max(t // 25, 1)):
        for j in range(top):
            e = int(idx[i, j])
            if e < 0:
                continue
            x = h[i].to(F)
            want = w2[e].to(F) @ (P.silu(w13[e, 0].to(F) @ x) * (w13[e, 1].to(F) @ x))
            assert err(got[i, j][None], want[None]) < 1.5 * TOL[dtype]


@BOTH
def test_embedding_feedback(dtype):
    w = rand(50, 72, dtype=torch.bfloat16)
    ids = torch.zeros(3, dtype=torch.int32, device=DEV)
    feedback = torch.tensor([4, 9, 49, 0], dtype=torch.int32, device=DEV)
    slots = torch.tensor([2, 0, 1], dtype=torch.int32, device=DEV)
    x, act = O.embed_residual(ids, w.to(DEV), dtype, feedback, slots, True)
    assert ids.tolist() == [49, 4, 9]
    assert torch.equal(x.cpu(), w[[49, 4, 9]].float()) and torch.equal(act.cpu(), w[[49, 4, 9]].to(dtype))
