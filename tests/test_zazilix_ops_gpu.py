"""The kernels of mixed residual streams, attention on chunks, gated linear attention and mixtures with inputs passed on, one
mechanism at a time, against the plain statements in ``plain_zazilix``."""
import math

import pytest
import torch

import plain_zazilix as P
from layered_checks import rel_err as err
from layered_util import make_fb
from minisgl.models.buvalix_weight import interleave_gate
from minisgl.ops import api as O
from minisgl.ops import cuda_gla as G
from minisgl.ops import cuda_mixers as C

pytestmark = pytest.mark.gpu
DEV = "cuda"
F = torch.float64
TOL = {torch.bfloat16: 1.2e-2, torch.float32: 2e-5}
BOTH = pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])


def rand(*shape, seed=0, std=1.0, mean=0.0, dtype=torch.float32):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * std + mean).to(dtype)


def on(x):
    return None if x is None else x.to(DEV)


# --------------------------------------------------------------------------- embedding, streams
@BOTH
@pytest.mark.parametrize("d,streams", [(96, 3), (50, 1), (2048, 4), (33, None), (64, None)])
def test_embedding_with_positions(d, streams, dtype):
    w, table = rand(40, d, dtype=torch.bfloat16), rand(90, d, seed=1, dtype=torch.bfloat16)
    ids, pos = torch.tensor([3, 0, 39, 3, 7], dtype=torch.int32), torch.tensor([0, 1, 89, 88, 5], dtype=torch.int32)
    x, act = O.embed_residual(on(ids), on(w), dtype, want_act=True, mul=1.75, table=on(table), positions=on(pos), streams=streams)
    want = w.to(F)[ids.long()] * 1.75 + table.to(F)[pos.long()]
    assert x.dtype == torch.float32 and err(act, want) < TOL[dtype]
    for s in ([x] if streams is None else x.unbind(1)):
        assert err(s, want) < 1e-6
    feedback, slots = torch.tensor([5, 0, 11, 2], dtype=torch.int32), torch.tensor([2, 0, 1, 2, 3], dtype=torch.int32)
    got_ids = on(ids)
    x, _ = O.embed_residual(got_ids, on(w), dtype, on(feedback), on(slots), streams=2)
    assert got_ids.tolist() == [11, 5, 0, 11, 2] and err(x[:, 1], w.to(F)[got_ids.cpu().long()]) < 1e-6


def plain_norm(u, eps, gain):
    return P.rms(u, eps) * gain


@BOTH
@pytest.mark.parametrize("d,s", [(96, 1), (100, 2), (1500, 3), (4096, 4), (33, 5), (2048, 4), (64, 16), (9000, 2), (8192, 3), (4096, 7)])
def test_streams(d, s, dtype):
    t, eps, k, n = 6, 1e-3, 4, 3
    x, sub, h = rand(t, s, d, mean=0.5), rand(t, d, seed=1), rand(t, d, seed=2).to(dtype)
    out, mix, pre, gain = rand(s, seed=3), rand(s, s, seed=4, std=0.5), rand(s, seed=5), 0.7
    post, pre_t = torch.cat([out, mix.reshape(-1)]), torch.cat([pre, torch.tensor([gain])])
    streams = x.to(F).transpose(0, 1)
    xd = on(x)
    got = O.stream_norm(xd, eps, dtype, pre=on(pre_t))
    assert torch.equal(xd.cpu(), x) and got.dtype == dtype
    assert err(got, plain_norm(P.stream_in(streams, pre.to(F)), eps, gain)) < TOL[dtype]
    # a projection's output comes in
    want = P.stream_out(streams, mix.to(F), out.to(F), sub.to(F))
    rows = torch.tensor([4, 0, 4])
    got = O.stream_norm(xd, eps, dtype, pre=on(pre_t), post=on(post), sub=on(sub), rows=on(rows))
    assert torch.equal(xd.cpu(), x) and err(got, plain_norm(P.stream_in(want, pre.to(F)), eps, gain)[rows]) < TOL[dtype]
    got = O.stream_norm(xd, eps, dtype, pre=on(pre_t), post=on(post), sub=on(sub), keep=False)
    assert torch.equal(xd.cpu(), x)
    got = O.stream_norm(xd, eps, dtype, pre=on(pre_t), post=on(post), sub=on(sub))
    assert err(xd.transpose(0, 1).reshape(s * t, d), want.reshape(s * t, d)) < 2e-6
    assert err(got, plain_norm(P.stream_in(want, pre.to(F)), eps, gain)) < TOL[dtype]
    # experts beside it: real ones, the input itself, none
    idx = torch.randint(-1, n + 2, (t, k), generator=torch.Generator().manual_seed(7)).to(torch.int32)
    idx[0] = torch.tensor([0, n, n + 1, 2])
    wts, rows_e = rand(t, k, seed=8), rand(t * k, d, seed=9).to(dtype)
    rows_e[idx.reshape(-1) < 0] = float("nan")
    rows_e[idx.reshape(-1) >= n] = float("nan")           # rows that no expert wrote
    y = sub.to(F).clone()
    for i in range(t):
        for j in range(k):
            if idx[i, j] >= 0:
                y[i] += wts[i, j].to(F) * (rows_e[i * k + j] if idx[i, j] < n else h[i]).to(F)
    for with_sub in (True, False):
        xd = on(x)
        got = O.stream_norm(xd, eps, dtype, pre=on(pre_t), post=on(post), sub=on(sub) if with_sub else None,
                            experts=(on(rows_e), on(wts), on(idx), n, on(h)))
        want = P.stream_out(streams, mix.to(F), out.to(F), y if with_sub else y - sub.to(F))
        assert err(xd.transpose(0, 1).reshape(s * t, d), want.reshape(s * t, d)) < 2e-6
        assert err(got, plain_norm(P.stream_in(want, pre.to(F)), eps, gain)) < TOL[dtype]
    assert O.stream_norm(xd, eps, dtype, post=on(post), sub=on(sub)) is None


# --------------------------------------------------------------------------- gated projection, router, experts
@BOTH
@pytest.mark.parametrize("t,d,f", [(5, 96, 40), (130, 72, 33), (1, 20, 7), (64, 1024, 320), (3000, 128, 1100), (1, 2048, 48)])
def test_silu_gated_projection(t, d, f, dtype):
    h = rand(t, d).to(dtype)
    g, u = (rand(f, d, seed=s, std=1.5 * d ** -0.5, dtype=torch.bfloat16) for s in (1, 2))
    got = O.gated_linear(on(h), on(interleave_gate(g, u)), "silu")
    x = h.to(F)
    want = P.silu(x @ g.to(F).T) * (x @ u.to(F).T)
    assert got.shape == (t, -(-f // 16) * 16) and float(got[:, f:].abs().max() if f % 16 else 0) == 0
    assert err(got[:, :f], want) < TOL[dtype]


@BOTH
@pytest.mark.parametrize("experts,top", [(12, 4), (3, 3), (70, 9), (512, 16), (1, 1)])
def test_router_over_all_outputs(experts, top, dtype):
    t, d, scale = 9, 128, 2.3
    h, w, b = rand(t, d).to(dtype), rand(experts, d, seed=1, std=2.0 * d ** -0.5, dtype=torch.bfloat16), rand(experts, seed=2, std=0.05)
    valid = torch.tensor([t - 1], dtype=torch.int32)
    idx, wts = O.route_topk(on(h), on(w), on(b), top, on(valid), "softmax", scale)
    s = torch.softmax(h.to(F) @ w.to(F).T, -1)
    chosen, weights = P.choose(h.to(F) @ w.to(F).T, b.to(F), top, scale)
    assert (idx[-1] == -1).all() and (wts[-1] == 0).all()
    idx, wts = idx.cpu().long()[:-1], wts.cpu()[:-1]
    key = (s + b.to(F))[:-1]
    # the same choice up to near ties, weights without the correction and not renormalised
    assert float((key.gather(1, idx) - key.gather(1, chosen[:-1])).abs().max()) < 1e-5
    assert err(wts, s[:-1].gather(1, idx) * scale) < 1e-4


def test_router_correction_changes_the_choice_and_not_the_weights():
    h, w = rand(4, 32), rand(6, 32, seed=1, dtype=torch.bfloat16)
    b = torch.tensor([0.0, 0.0, 5.0, 0.0, 4.0, 0.0])
    idx, wts = O.route_topk(on(h), on(w), on(b), 2, None, "softmax", 3.0)
    s = torch.softmax(h.to(F) @ w.to(F).T, -1)
    assert (idx.cpu() == torch.tensor([2, 4])).all() and err(wts, s[:, [2, 4]] * 3.0) < 1e-4


@BOTH
@pytest.mark.parametrize("t,d,f,experts,identity,top", [(7, 96, 40, 5, 3, 4), (70, 64, 128, 4, 2, 3), (3, 50, 21, 2, 1, 3), (300, 128, 64, 8, 0, 2)])
def test_experts_beside_identities(t, d, f, experts, identity, top, dtype):
    """Router, experts, identities, shared expert and the streams' update together."""
    h = rand(t, d).to(dtype)
    p = {"router": rand(experts + identity, d, seed=1, std=3.0 * d ** -0.5), "correction": rand(experts + identity, seed=2, std=0.02)}
    for e, name in enumerate([f"e{e}" for e in range(experts)] + ["shared"]):
        p[name + ".gate"], p[name + ".up"] = (rand(f, d, seed=10 + 3 * e + i, std=d ** -0.5) for i in (0, 1))
        p[name + ".down"] = rand(d, f, seed=12 + 3 * e, std=f ** -0.5)
    p = {k: v if k == "correction" else v.bfloat16() for k, v in p.items()}
    w13 = torch.stack([torch.stack([p[f"e{e}.gate"], p[f"e{e}.up"]]) for e in range(experts)])
    w2 = torch.stack([p[f"e{e}.down"] for e in range(experts)])
    idx, wts = O.route_topk(on(h), on(p["router"]), on(p["correction"]), top, None, "softmax", 1.9)
    rows = O.gated_experts(on(h), idx, wts, on(w13), on(w2))
    x = torch.zeros(t, 1, d, device=DEV)
    O.stream_norm(x, 1e-5, dtype, post=torch.tensor([1.0, 0.0], device=DEV), sub=torch.zeros(t, d, device=DEV),
                  experts=(rows, wts, idx, experts, on(h)))
    pd = {k: v.to(F) for k, v in p.items()}
    hd = h.to(F)
    want = torch.zeros(t, d, dtype=F)
    ids, s = idx.cpu().long(), torch.softmax(hd @ pd["router"].T, -1)
    for i in range(t):
        for e in ids[i].tolist():
            want[i] += 1.9 * s[i, e] * (P.gated(hd[i:i + 1], pd, f"e{e}")[0] if e < experts else hd[i])
    if identity:
        assert int((ids >= experts).sum()) > 0
    assert err(x[:, 0], want) < 3 * TOL[dtype]


# --------------------------------------------------------------------------- norms ahead of the cache
@BOTH
@pytest.mark.parametrize("heads,kv,dim,vdim,rot", [(4, 2, 24, 40, 0), (3, 1, 10, 14, 0), (16, 4, 128, 128, 0), (6, 3, 16, 8, 8), (3, 3, 7, 9, 6)])
def test_norms_over_the_whole_projection(heads, kv, dim, vdim, rot, dtype):
    fb, rows = make_fb([(1, 0, 5), (2, 22, 4), (0, 300, 2)], DEV)
    t, n, eps = 11, (heads + kv) * dim + kv * vdim, 1e-2
    wide = rand(t, n + 8, std=0.3).to(dtype)          # a column slice of a wider projection
    gain = rand((heads + kv) * dim, seed=1, mean=1.0)
    freq = torch.tensor([700.0 ** (-2.0 * i / rot) for i in range(rot // 2)]) if rot else None
    keys, values = (torch.zeros(rows, kv * w, dtype=dtype, device=DEV) for w in (dim, vdim))
    got = O.rotate_store(on(wide)[:, :n], None, on(freq), None, keys, values, fb, heads, kv, dim, vdim, on(gain), True, eps, 0.6)
    q, k, v = wide[:, :n].to(F).split([heads * dim, kv * dim, kv * vdim], 1)
    q, k = P.rms(q, eps) * gain[:heads * dim].to(F), P.rms(k, eps) * gain[heads * dim:].to(F)
    v = 0.6 * P.rms(v.reshape(t, kv, vdim), eps).reshape(t, -1)
    if rot:
        import plain_buvalix as B

        pos = fb.positions.cpu()
        q = B.rotate(q.reshape(t, heads, dim), pos, rot, 700.0).reshape(t, -1)
        k = B.rotate(k.reshape(t, kv, dim), pos, rot, 700.0).reshape(t, -1)
    loc = fb.out_loc.cpu().long()
    assert err(got.flatten(1), q) < TOL[dtype] and err(keys[on(loc)], k) < TOL[dtype] and err(values[on(loc)], v) < TOL[dtype]


# --------------------------------------------------------------------------- attention on chunks
def attention_case(heads, kv, dim, vdim, size, segs, dtype, prefill=True, scale=0.2, edit=None, seed=0, max_len=2048):
    fb, rows = make_fb(segs, DEV, prefill=prefill, max_len=max_len)
    t = sum(n for _, _, n in segs)
    q, keys, values = rand(t, heads, dim, seed=seed + 1), rand(rows, kv * dim, seed=seed + 2), rand(rows, kv * vdim, seed=seed + 3)
    if edit:
        edit(q, keys, values, fb)
    q, keys, values = q.to(dtype), keys.to(dtype), values.to(dtype)
    slope = torch.tensor(P.slopes(heads))
    got = O.grouped_attention(on(q), on(keys), on(values), fb, kv, scale, 0.0, torch.zeros(heads, device=DEV), None, on(slope), size)
    want, at = [], 0
    table = fb.page_table.cpu()
    for slot, a, n in segs:
        loc = table[slot, :a + n].long()
        want.append(P.chunk_attend(q[at:at + n].to(F), keys[loc].to(F).view(a + n, kv, dim), values[loc].to(F).view(a + n, kv, vdim),
                                   scale, size).reshape(n, -1))
        at += n
    return got, torch.cat(want)


SHAPES = [(4, 2, 24, 40), (3, 1, 10, 14), (16, 4, 64, 64), (20, 1, 128, 96), (2, 2, 160, 144)]


@BOTH
@pytest.mark.parametrize("heads,kv,dim,vdim", SHAPES)
@pytest.mark.parametrize("size", [1, 37, 64, 100, 5000])
def test_prefill_on_chunks(heads, kv, dim, vdim, size, dtype):
    segs = [(1, 0, 90), (2, 35, 4), (3, 99, 2), (0, 60, 130), (4, 128, 1)]
    got, want = attention_case(heads, kv, dim, vdim, size, segs, dtype)
    assert err(got, want) < 1.5 * TOL[dtype]


@pytest.mark.parametrize("form", ["flash", "rows", "auto"])
@pytest.mark.parametrize("size", [50, 64, 200, 333, 1000])
def test_every_kernel_of_prefill_on_chunks(form, size, monkeypatch):
    """Long portions that begin and end anywhere in a chunk, page or key tile."""
    monkeypatch.setattr(C, "GROUPED_PREFILL", form)
    segs = [(1, 0, 600), (2, 190, 30), (3, 199, 70), (0, 130, 300), (4, 1000, 2)]
    got, want = attention_case(6, 3, 40, 48, size, segs, torch.bfloat16)
    assert err(got, want) < 1.5 * TOL[torch.bfloat16]


@BOTH
@pytest.mark.parametrize("heads,kv,dim,vdim", SHAPES)
@pytest.mark.parametrize("size", [1, 37, 64, 700])
def test_decode_on_chunks(heads, kv, dim, vdim, size, dtype):
    segs = [(0, 0, 1), (1, 36, 1), (2, 37, 1), (3, 63, 1), (4, 64, 1), (5, 699, 1)]
    got, want = attention_case(heads, kv, dim, vdim, size, segs, dtype, prefill=False)
    assert err(got, want) < 1.5 * TOL[dtype]


@BOTH
@pytest.mark.parametrize("portion", [1, 2, 40, 150])
@pytest.mark.parametrize("size", [48, 128])
def test_a_key_just_inside_and_just_outside_a_chunk(size, portion, dtype):
    """One key answers every query loudly; it stands at the first place of a chunk, or at the last of the one before."""
    start = 3 * size - portion // 2
    for at in (2 * size, 3 * size, 2 * size - 1, 3 * size - 1):
        def edit(q, keys, values, fb):
            q[:] = q.abs() + 1.0
            loc = int(fb.page_table[1, at])
            keys[loc], values[loc] = 4.0, 50.0

        segs = [(1, start, portion)]
        got, want = attention_case(4, 2, 16, 16, size, segs, dtype, prefill=portion > 1, edit=edit)
        assert err(got, want) < 2 * TOL[dtype]
        seen = [i // size == at // size and i >= at for i in range(start, start + portion)]
        loud = (want.abs().amax(-1) > 20).tolist()
        assert all(s or not l for s, l in zip(seen, loud)) and (not any(seen) or any(loud))


def test_slope_far_away_and_the_added_one():
    """Equal scores: the weights are a geometric series in the distance, next to the one in the denominator."""
    heads, n = 8, 600
    fb, rows = make_fb([(1, n - 1, 1)], DEV, prefill=False)
    q, keys = torch.zeros(1, heads, 16, device=DEV), torch.zeros(rows, 16, device=DEV)
    values = torch.zeros(rows, 16, device=DEV)
    place = torch.arange(n, dtype=torch.float32, device=DEV)
    values[fb.page_table[1, :n].long()] = place[:, None]
    got = O.grouped_attention(q, keys, values, fb, 1, 1.0, 0.0, torch.zeros(heads, device=DEV), None, torch.tensor(P.slopes(heads), device=DEV), 0)
    for h, m in enumerate(P.slopes(heads)):
        w = torch.exp(-m * (n - 1 - place.cpu().to(F)))
        assert math.isclose(float(got.view(heads, 16)[h, 0]), float((w * place.cpu()).sum() / (1 + w.sum())), rel_tol=2e-5), h


# --------------------------------------------------------------------------- gates with a running maximum
@pytest.mark.parametrize("segs", [[(1, 0, 1), (2, 5, 1)], [(1, 0, 70), (3, 40, 2), (2, 9, 33)], [(0, 0, 1500), (4, 100, 300)]])
@pytest.mark.parametrize("cap,gain", [(8.0, 2.0), (30.0, 20.0)])
def test_gates_with_a_running_maximum(segs, cap, gain):
    heads, (fb, _) = 5, make_fb(segs, DEV, prefill=max(n for _, _, n in segs) > 1)
    t = sum(n for _, _, n in segs)
    z, b, top = rand(t, 2 * heads, std=gain), rand(2 * heads, seed=1) + 1.0, rand(7, heads, seed=2, std=3.0)
    topd = on(top)
    log_g, fac, floor = (x.cpu().to(F) for x in O.mlstm_gates(on(z), on(b), cap, topd, fb))
    g = cap * torch.tanh((z.to(F) + b.to(F)) / cap)
    i, f, at = g[:, :heads], P.log_sigmoid(g[:, heads:]), 0
    for slot, a, n in segs:
        m = top[slot].to(F) if a else torch.zeros(heads, dtype=F)
        for r in range(at, at + n):
            new = torch.maximum(f[r] + m, i[r])
            assert torch.allclose(log_g[r], f[r] + m - new, atol=3e-5) and torch.allclose(fac[r], torch.exp(i[r] - new), rtol=5e-5, atol=1e-30)
            assert torch.allclose(floor[r], torch.exp(-new), rtol=5e-5)
            m = new
        assert torch.allclose(topd[slot].cpu().to(F), m, atol=3e-5)
        at += n
    untouched = [s for s in range(7) if s not in [s for s, _, _ in segs]]
    assert torch.equal(topd[untouched].cpu(), top[untouched])


# --------------------------------------------------------------------------- short convolution
@BOTH
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
@pytest.mark.parametrize("c", [48, 30, 700])
def test_causal_convolution(c, taps, dtype):
    segs = [(1, 0, 1), (2, 9, 1), (3, 0, 40), (4, 3, 2), (0, 17, 33)]
    for prefill in (True, False):
        part = segs if prefill else segs[:2]
        fb, _ = make_fb(part, DEV, prefill=prefill)
        t = sum(n for _, _, n in part)
        p, w, b = rand(t, c + 16).to(dtype), rand(taps, c, seed=1), rand(c, seed=2)
        before = rand(7, taps - 1, c, seed=3).to(dtype)
        bd = on(before)
        got, at = O.causal_conv(on(p)[:, 8:8 + c], on(w), on(b), bd, fb), 0
        for slot, a, n in part:
            old = before[slot].to(F) if a else torch.zeros(taps - 1, c, dtype=F)
            y, keep = P.short_conv(p[at:at + n, 8:8 + c].to(F), w.to(F).T, b.to(F), old)
            assert err(got[at:at + n], y) < TOL[dtype]
            if taps > 1:
                assert torch.equal(bd[slot].cpu(), keep.to(dtype))
            at += n
        untouched = [s for s in range(7) if s not in [s for s, _, _ in part]]
        assert torch.equal(bd[untouched].cpu(), before[untouched])


# --------------------------------------------------------------------------- the recurrences
def gla_case(kind, heads, groups, d, e, segs, dtype, speed=0.0, prefill=True, seed=0, q_mul=1.0):
    """(got, want, got states, want states) of one recurrence; speed: shift of the decays' logits."""
    fb, _ = make_fb(segs, DEV, prefill=prefill)
    t = sum(n for _, _, n in segs)
    cols = -(-(e + (kind == "given")) // 4) * 4
    pq, pk, pv = (rand(t, n + 16, seed=seed + i).to(dtype)[:, 8:8 + n] for i, n in enumerate((groups * d, groups * d, heads * e)))
    state = rand(7, heads, d, cols, seed=seed + 3)
    if kind == "given":
        gates = (-torch.exp(rand(t, heads, seed=seed + 4) + speed), torch.exp(rand(t, heads, seed=seed + 5) - 1))
    elif kind == "step":
        gates = (rand(t, heads, seed=seed + 4) + speed, rand(heads, seed=seed + 5) - 1, rand(heads, seed=seed + 6))
    else:
        gates = (rand(t, heads * d, seed=seed + 4) - speed, rand(heads * d, seed=seed + 5) + 1, rand(heads * d, seed=seed + 6).sigmoid() * 0.8)
        if speed > 5:
            gates = (gates[0], gates[1], gates[2] * 0)
    sd = on(state)
    wide = lambda x: torch.nn.functional.pad(x, (8, 8)).to(DEV)[:, 8:-8]
    got = O.gla(kind, wide(pq), None if kind == "forget" else wide(pk), wide(pv), tuple(on(g) for g in gates), sd, fb, heads, groups, q_mul)
    spread = lambda x: x.to(F).reshape(t, groups, d).repeat_interleave(heads // groups, 1)
    q, k, v = spread(pq), spread(pk), pv.to(F).reshape(t, heads, e)
    gd = [g.to(F) for g in gates]
    want, states, at = [], [], 0
    for slot, a, n in segs:
        r = slice(at, at + n)
        s = state[slot].to(F) if a else torch.zeros(heads, d, cols, dtype=F)
        if kind == "given":
            ones = torch.cat([v[r], torch.ones(n, heads, 1, dtype=F)], -1)
            f = torch.exp(gd[0][r])[..., None].expand(n, heads, d)
            o, s2 = [], s[..., :e + 1]
            for i in range(n):
                s2 = f[i][:, :, None] * s2 + gd[1][r][i][:, None, None] * k[r][i][:, :, None] * ones[i][:, None, :]
                o.append((s2 * q[r][i][:, :, None]).sum(1) * q_mul)
            o = torch.stack(o)
        elif kind == "step":
            dt = P.softplus(gd[0][r] + gd[1])
            o, s2 = P.mamba_recurrence(v[r], k[r], q[r] * q_mul, dt, gd[2], torch.zeros(heads, dtype=F), s[..., :e])
        else:
            f = gd[2] + (1 - gd[2]) * P.sigmoid(gd[0][r] + gd[1])
            o, s2 = P.hgrn_recurrence(P.silu(q[r]) * q_mul, f.view(n, heads, d), v[r], s[..., :e])
        want.append(o)
        states.append(s2)
        at += n
    n = want[0].shape[-1]
    got_states = torch.stack([sd[s][..., :n] for s, _, _ in segs])
    untouched = [s for s in range(7) if s not in [s for s, _, _ in segs]]
    assert torch.equal(sd[untouched].cpu(), state[untouched])
    return got[..., :n].flatten(1), torch.cat(want).flatten(1), got_states.flatten(1), torch.stack(states).flatten(1)


KINDS = pytest.mark.parametrize("kind", ["given", "step", "forget"])
SIZES = [(3, 3, 24, 16), (4, 2, 16, 40), (2, 1, 64, 64), (2, 2, 128, 128), (1, 1, 9, 7), (2, 1, 200, 264), (1, 1, 1, 1), (2, 2, 40, 136)]


def gla_sizes(kind, groups, heads):
    return heads if kind != "step" else groups


@KINDS
@BOTH
@pytest.mark.parametrize("heads,groups,d,e", SIZES)
def test_recurrence_token_by_token(kind, heads, groups, d, e, dtype, monkeypatch):
    monkeypatch.setattr(G, "GLA_CHUNKED", False)
    g = gla_sizes(kind, groups, heads)
    got, want, s, ws = gla_case(kind, heads, g, d, e, [(1, 0, 20), (2, 7, 9), (4, 1, 1)], dtype, q_mul=d ** -0.5)
    assert err(got, want) < 1e-4 and err(s, ws) < 1e-5
    got, want, s, ws = gla_case(kind, heads, g, d, e, [(1, 0, 1), (2, 7, 1), (5, 99, 1)], dtype, prefill=False)
    assert err(got, want) < 1e-4 and err(s, ws) < 1e-5


@KINDS
@pytest.mark.parametrize("heads,groups,d,e", [(3, 3, 24, 16), (4, 2, 16, 40), (2, 1, 64, 64), (2, 2, 128, 128), (2, 1, 48, 264), (1, 1, 8, 8)])
@pytest.mark.parametrize("segs", [[(1, 0, 64)], [(1, 0, 200), (2, 70, 65), (0, 3, 1), (5, 0, 2), (3, 63, 130)]])
def test_recurrence_in_chunks(kind, heads, groups, d, e, segs):
    """Portions that fill no chunk, states that go on; bf16 activations, 32-bit everything else."""
    got, want, s, ws = gla_case(kind, heads, gla_sizes(kind, groups, heads), d, e, segs, torch.bfloat16, speed=-2.0, q_mul=d ** -0.5)
    assert err(got, want) < 2e-4 and err(s, ws) < 2e-5


@KINDS
@pytest.mark.parametrize("speed", [-12.0, -6.0, 0.0, 3.0, 8.0, 40.0])
def test_chunks_with_slow_and_fast_decays(kind, speed):
    """From decays that hardly forget over hundreds of tokens to ones that clear the state at once (per channel: exponents that no
    block of tokens can hold).  Running sums of logs that reach thousands are good to 1e-4."""
    speed = min(speed, 3.0) if kind == "given" else speed
    got, want, s, ws = gla_case(kind, 2, 1 if kind == "step" else 2, 32, 24, [(1, 0, 300), (2, 5, 64)], torch.bfloat16, speed=speed)
    assert err(got, want) < 5e-4 and err(s, ws) < 5e-4


@KINDS
def test_a_far_token_in_a_recurrence(kind):
    """The first token's key answers the last queries only; hardly anything is forgotten."""
    for dtype in (torch.bfloat16, torch.float32):
        got, want, _, _ = gla_case(kind, 2, 1 if kind == "step" else 2, 16, 16, [(1, 0, 500)], dtype, speed=-9.0, seed=3)
        assert err(got[-5:], want[-5:]) < 2e-4


def test_padded_rows_leave_the_state_alone():
    fb, _ = make_fb([(1, 4, 1), (2, 8, 1), (3, 2, 1)], DEV, prefill=False)
    fb.num_valid = torch.tensor([2], dtype=torch.int32, device=DEV)
    state, top, before = rand(7, 2, 16, 20).to(DEV), rand(7, 2).to(DEV), rand(7, 2, 24).to(DEV)
    old = state.clone(), top.clone(), before.clone()
    gates = O.mlstm_gates(on(rand(3, 4)), on(rand(4)), 9.0, top, fb)
    O.gla("given", *(on(rand(3, 32, seed=i)) for i in range(3)), gates[:2], state, fb, 2, 2)
    O.causal_conv(on(rand(3, 24)), on(rand(3, 24)), on(rand(24)), before, fb)
    for new, was in zip((state, top, before), old):
        assert torch.equal(new[3], was[3]) and not torch.equal(new[1], was[1]) and not torch.equal(new[2], was[2])


# --------------------------------------------------------------------------- behind the recurrences
@BOTH
@pytest.mark.parametrize("heads,e", [(3, 16), (2, 7), (4, 128), (1, 300), (2, 2), (16, 64)])
def test_norms_of_heads(heads, e, dtype):
    t, eps = 9, 1e-3
    ew = -(-(e + 1) // 4) * 4
    o, floor = rand(t, heads, ew, std=0.1), rand(t, heads, seed=1).abs() * 0.1
    o[..., e + 1:] = float("nan")
    gate, gain, own = rand(t, heads * e + 8, seed=2).to(dtype)[:, :heads * e], rand(heads * e, seed=3), rand(e, seed=4)
    x = o[..., :e].to(F)
    got = O.norm_heads(on(o), e, on(own), eps, dtype, mul=0.4)
    assert err(got, (P.rms(x, eps) * own.to(F) * 0.4).reshape(t, -1)) < TOL[dtype]
    y = x / (torch.maximum(o[..., e].to(F).abs(), floor.to(F)) + 1e-6)[..., None]
    want = P.rms(y, eps).reshape(t, -1) * gain.to(F) * P.sigmoid(gate.to(F))
    got = O.norm_heads(on(o), e, on(gain), eps, dtype, gate=torch.nn.functional.pad(gate, (0, 8)).to(DEV)[:, :heads * e], floor=on(floor))
    assert err(got, want) < TOL[dtype]


@BOTH
@pytest.mark.parametrize("heads,e,groups", [(4, 24, 2), (3, 7, 3), (64, 64, 1), (6, 16, 12), (2, 5, 10), (80, 64, 8), (96, 96, 1)])
def test_norms_of_groups(heads, e, groups, dtype):
    """Groups within a head, over several heads, across the heads' borders."""
    t, eps, n = 5, 1e-3, heads * e
    ew = -(-e // 4) * 4
    o, skip, gain = rand(t, heads, ew), rand(heads, seed=1), rand(n, seed=2)
    x, z = (rand(t, n + 24, seed=s).to(dtype) for s in (3, 4))
    got = O.norm_groups(on(o), on(skip), on(x)[:, 8:8 + n], on(z)[:, 16:16 + n], on(gain), groups, eps)
    y = (o[..., :e].to(F) + skip.to(F)[:, None] * x[:, 8:8 + n].to(F).reshape(t, heads, e)).reshape(t, n)
    y = y * P.silu(z[:, 16:16 + n].to(F))
    assert err(got, P.rms(y.view(t, groups, -1), eps).reshape(t, n) * gain.to(F)) < TOL[dtype]
