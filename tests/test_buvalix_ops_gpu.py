"""The kernels of layer norms, gated projections, grouped attention and the gated delta rule, one mechanism at a time, against
the plain statements in ``plain_buvalix``."""
import math

import pytest
import torch

import plain_buvalix as P
from layered_util import make_fb
from minisgl.models.buvalix_weight import interleave_gate, spread_buckets
from minisgl.ops import api as O
from minisgl.ops import cuda_mixers as C

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
@pytest.mark.parametrize("d", [96, 100, 1500, 4096, 9000, 33])
def test_residual_layer_norm(d, dtype):
    n, eps = 7, 1e-3
    x, y, add = rand(n, d) + 3.0, rand(n, d, seed=1) * 2 - 1, rand(n, d, seed=2).to(dtype)
    w1, b1, w2, b2 = (rand(d, seed=s) for s in (3, 4, 5, 6))
    dev = [t.to(DEV) for t in (w1, b1, w2, b2)]
    want = x.to(F) + P.layer_norm(y.to(F), w1.to(F), b1.to(F), eps)
    xc = x.to(DEV)
    h = O.residual_layer_norm(xc, eps, dtype, norm=dev[2:], sub=(y.to(DEV), *dev[:2]))
    assert err(xc, want) < 1e-6 and h.dtype == dtype
    assert err(h, P.layer_norm(want, w2.to(F), b2.to(F), eps)) < TOL[dtype]
    want = want + add.to(F)
    h = O.residual_layer_norm(xc, eps, dtype, norm=dev[2:], add=add.to(DEV))
    assert err(xc, want) < 1e-6 and err(h, P.layer_norm(want, w2.to(F), b2.to(F), eps)) < TOL[dtype]
    before, pick = xc.clone(), torch.tensor([5, 0, 5])
    h = O.residual_layer_norm(xc, eps, dtype, norm=dev[2:], sub=(y.to(DEV), *dev[:2]), rows=pick.to(DEV))
    more = want + P.layer_norm(y.to(F), w1.to(F), b1.to(F), eps)
    assert torch.equal(xc, before) and err(h, P.layer_norm(more, w2.to(F), b2.to(F), eps)[pick]) < TOL[dtype]
    h = O.residual_layer_norm(xc, eps, dtype, norm=dev[2:])
    assert torch.equal(xc, before) and err(h, P.layer_norm(want, w2.to(F), b2.to(F), eps)) < TOL[dtype]
    assert O.residual_layer_norm(xc, eps, dtype, sub=(y.to(DEV), *dev[:2])) is None
    assert err(xc, more) < 1e-6


def test_layer_norm_of_a_row_far_from_zero():
    """The deviations are taken from the mean, not from the difference of two large squares."""
    x, d = rand(3, 512, std=1e-2) + 100.0, 512
    got = O.residual_layer_norm(x.to(DEV), 1e-6, torch.float32, norm=(torch.ones(d, device=DEV), torch.zeros(d, device=DEV)))
    assert err(got, P.layer_norm(x.to(F), 1.0, 0.0, 1e-6)) < 1e-3


# --------------------------------------------------------------------------- gated projection
@BOTH
@pytest.mark.parametrize("t,d,f", [(5, 96, 40), (130, 72, 33), (1, 20, 7), (64, 1024, 320), (300, 264, 520), (3000, 128, 1100),
                                   (1, 2048, 48), (140, 64, 6000)])
def test_gated_projection(t, d, f, dtype):
    """Every tile width, split sums, the persistent kernel, rows that TMA cannot fetch, sizes padded to blocks of 16."""
    h = rand(t, d).to(dtype)
    g, u = (rand(f, d, seed=s, std=1.5 * d ** -0.5, dtype=torch.bfloat16) for s in (1, 2))
    got = O.gated_linear(h.to(DEV), interleave_gate(g, u).to(DEV), "gelu_tanh")
    x = h.to(F)
    want = P.gelu_tanh(x @ g.to(F).T) * (x @ u.to(F).T)
    assert got.shape == (t, -(-f // 16) * 16) and float(got[:, f:].abs().max() if f % 16 else 0) == 0
    assert err(got[:, :f], want) < TOL[dtype]


def test_gelu_far_from_zero():
    z = torch.tensor([[-40.0, -8.0, -3.0, -1e-3, 0.0, 1e-3, 3.0, 30.0] * 4], dtype=torch.float32)
    eye = torch.eye(32, dtype=torch.bfloat16)
    got = O.gated_linear(z.to(DEV), interleave_gate(eye, eye).to(DEV), "gelu_tanh")
    zd = z.to(F)
    assert torch.allclose(got.cpu().to(F), P.gelu_tanh(zd) * zd, rtol=1e-5, atol=1e-6)


# --------------------------------------------------------------------------- rotation, temperature, cache rows
@BOTH
@pytest.mark.parametrize("heads,kv,dim,vdim,rot,temp,bias", [(4, 2, 24, 40, 16, None, True), (3, 1, 10, 14, 10, None, True),
                                                             (6, 3, 16, 8, 0, (0.4, 24), False), (2, 2, 64, 32, 64, (0.2, 1), True),
                                                             (16, 4, 128, 128, 2, None, False), (1, 1, 7, 9, 6, (1.5, 7), False)])
def test_rotate_store(heads, kv, dim, vdim, rot, temp, bias, dtype):
    segs = [(1, 0, 5), (2, 22, 4), (3, 1023, 1), (0, 9000, 2)]
    fb, rows = make_fb(segs, DEV, max_len=9100)
    fb.out_loc[3] = -1
    t, n = 12, (heads + kv) * dim + kv * vdim
    wide = rand(t, n + 8 if n % 8 == 0 else n + 3).to(dtype)
    b = rand(n, seed=1) if bias else None
    freq = (torch.tensor([5000.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=F).float()) if rot else None
    keys, values = (torch.full((rows, kv * w), 7.0, dtype=dtype, device=DEV) for w in (dim, vdim))
    on = lambda x: None if x is None else x.to(DEV)
    got = O.rotate_store(wide.to(DEV)[:, :n].contiguous(), on(b), on(freq), temp, keys, values, fb, heads, kv, dim, vdim)
    x = wide[:, :n].to(F) + (b.to(F) if bias else 0.0)
    q, k, v = x.split([heads * dim, kv * dim, kv * vdim], 1)
    pos = fb.positions.cpu()
    q, k = q.reshape(t, heads, dim), k.reshape(t, kv, dim)
    if rot:
        q, k = P.rotate(q, pos, rot, 5000.0), P.rotate(k, pos, rot, 5000.0)
    if temp:
        q = q * torch.tensor([P.query_temperature(int(p), *temp) for p in pos], dtype=F)[:, None, None]
    tol = max(TOL[dtype], 3e-4 if rot else 0.0)          # 32-bit angles of positions around 9 000
    assert err(got.flatten(1), q.flatten(1)) < tol
    assert err(got[:8].flatten(1), q[:8].flatten(1)) < max(TOL[dtype], 2e-5)
    loc = fb.out_loc.cpu().long()
    for i in range(t):
        if i != 3:
            assert err(keys[loc[i]][None], k[i].reshape(1, -1)) < tol and err(values[loc[i]][None], v[i][None]) < TOL[dtype]
    assert int((keys[:, 0] != 7.0).sum()) <= t - 1


# --------------------------------------------------------------------------- grouped attention
SEGS = [[(0, 0, 1)], [(1, 0, 70)], [(2, 63, 2), (0, 0, 5), (3, 200, 130)], [(4, 1000, 3), (1, 0, 200), (2, 15, 1)],
        [(1, 127, 129), (2, 128, 257), (3, 1, 255), (4, 500, 33), (0, 640, 1)]]


def attention_case(segs, heads, kv, dim, vdim, dtype, prefill=True, seed=0, std=1.0):
    fb, rows = make_fb(segs, DEV, seed=seed, prefill=prefill)
    t = fb.positions.shape[0]
    return (fb, rand(t, heads, dim, seed=seed, std=std).to(dtype), rand(rows, kv * dim, seed=seed + 1).to(dtype),
            rand(rows, kv * vdim, seed=seed + 2).to(dtype))


def plain_attention(q, keys, values, fb, kv, scale, cap, sink, rel, rows=None):
    """[rows, H * vdim] of the listed rows; rel: (table [buckets, H], limit)."""
    table, slots, pos = fb.page_table.cpu().long(), fb.slots.cpu().long(), fb.positions.cpu()
    heads, dim = q.shape[1:]
    out = []
    for i in rows if rows is not None else range(q.shape[0]):
        loc = table[slots[i], : int(pos[i]) + 1]
        k, v = keys[loc].to(F).view(len(loc), kv, dim), values[loc].to(F).view(len(loc), kv, -1)
        bias = None
        if rel is not None:
            buckets = torch.tensor([P.distance_bucket(n, rel[0].shape[0], rel[1]) for n in range(len(loc))])
            bias = lambda away: rel[0].to(F)[buckets[away]]
        out.append(P.attend(q[i:i + 1].to(F), k, v, heads // kv, scale, cap if cap else 1e9, None if sink is None else sink.to(F),
                            bias))
    return torch.cat(out).flatten(1)


def check_attention(segs, heads, kv, dim, vdim, dtype, cap, with_sink, rel, prefill=True, std=1.0, every=1, tol=None):
    fb, q, keys, values = attention_case(segs, heads, kv, dim, vdim, dtype, prefill, std=std)
    sink = rand(heads, seed=9) * 2 if with_sink else None
    scale = 1.3 / math.sqrt(dim)
    on = lambda x: None if x is None else x.to(DEV)
    table = None if rel is None else spread_buckets(*rel).to(DEV)
    got = O.grouped_attention(q.to(DEV), keys.to(DEV), values.to(DEV), fb, kv, scale, cap, on(sink), table)
    t = q.shape[0]
    rows = sorted(set(range(0, t, every)) | {t - 1, 0})
    want = plain_attention(q, keys, values, fb, kv, scale, cap, sink, rel, rows)
    per_head = lambda x: x.reshape(len(rows) * heads, vdim)
    assert err(per_head(got.cpu()[rows]), per_head(want)) < (tol or 2 * TOL[dtype])
    return got


SIZES = [(1, 1, 8, 8), (4, 2, 24, 40), (6, 2, 40, 48), (8, 1, 64, 128), (5, 5, 128, 72), (40, 2, 32, 64), (3, 1, 200, 136)]


@BOTH
@pytest.mark.parametrize("heads,kv,dim,vdim", SIZES + [(3, 3, 10, 14), (2, 1, 300, 40), (2, 2, 20, 260)])
@pytest.mark.parametrize("segs", SEGS[:4])
def test_prefill_with_cap_and_sink(heads, kv, dim, vdim, segs, dtype):
    check_attention(segs, heads, kv, dim, vdim, dtype, 5.0, True, None, every=7)


@BOTH
@pytest.mark.parametrize("heads,kv,dim,vdim", SIZES)
@pytest.mark.parametrize("segs", SEGS)
def test_prefill_with_cap_and_distance_bias(heads, kv, dim, vdim, segs, dtype):
    check_attention(segs, heads, kv, dim, vdim, dtype, 9.0, False, (rand(18, heads, seed=4) * 2, 150), every=11)


@pytest.mark.parametrize("form", ["flash", "rows"])
@pytest.mark.parametrize("cap,with_sink,rel", [(0.0, False, False), (0.0, True, True), (3.0, True, True), (4.0, False, False)])
@pytest.mark.parametrize("segs", SEGS)
def test_both_prefill_kernels_with_every_option(form, cap, with_sink, rel, segs, monkeypatch):
    monkeypatch.setattr(C, "GROUPED_PREFILL", form)
    table = (rand(32, 4, seed=5) * 2, 400) if rel else None
    check_attention(segs, 4, 2, 72, 56, torch.bfloat16, cap, with_sink, table, every=9)


@pytest.mark.parametrize("std", [0.1, 3.0, 30.0])
def test_small_and_large_scores_under_the_cap(std):
    """Scores well under the cap, around it, and saturated: both forms of the hyperbolic tangent."""
    for segs in ([(1, 0, 300)], [(2, 90, 3)]):
        check_attention(segs, 2, 1, 64, 64, torch.bfloat16, 6.0, True, None, std=std, every=13, tol=3e-2)
    check_attention([(1, 0, 100)], 2, 1, 64, 64, torch.float32, 6.0, True, None, std=std, every=13, tol=1e-4)


@BOTH
@pytest.mark.parametrize("heads,kv,dim,vdim", SIZES + [(128, 2, 64, 64)])
def test_decode(heads, kv, dim, vdim, dtype):
    """Single rows at, before and behind page and key-tile borders; with and without split keys."""
    segs = [(0, 0, 1), (1, 15, 1), (2, 16, 1), (3, 63, 1), (4, 64, 1), (5, 1700, 1)]
    a = check_attention(segs, heads, kv, dim, vdim, dtype, 7.0, True, (rand(20, heads, seed=4), 90), prefill=False)
    b = check_attention(segs, heads, kv, dim, vdim, dtype, 7.0, True, (rand(20, heads, seed=4), 90), prefill=True)
    assert err(a, b.cpu().to(F)) < TOL[dtype]


def test_padded_rows_are_left_alone():
    fb, q, keys, values = attention_case([(0, 5, 1), (1, 9, 1), (6, 0, 1), (6, 0, 1)], 4, 2, 64, 32, torch.bfloat16, False)
    fb.num_valid = torch.tensor([2], dtype=torch.int32, device=DEV)
    got = O.grouped_attention(q.to(DEV), keys.to(DEV), values.to(DEV), fb, 2, 0.1, 5.0)
    assert err(got[:2], plain_attention(q, keys, values, fb, 2, 0.1, 5.0, None, None)[:2]) < 1.2e-2


@BOTH
@pytest.mark.parametrize("far", [0, 1, 15, 16, 63, 64, 127, 128, 700])
@pytest.mark.parametrize("portion", [0, 9, 100, 300])
def test_one_key_stands_out(far, portion, dtype):
    """Queries that are almost a multiple of one far key: a key that is missed, or taken from a wrong page, shows."""
    n, heads, kv, dim = 701, 4, 2, 64
    fb, rows = make_fb([(2, n - max(portion, 1), max(portion, 1))], DEV, prefill=portion > 0)
    t = fb.positions.shape[0]
    keys, values = rand(rows, kv * dim, seed=3).to(dtype), rand(rows, kv * 32, seed=4).to(dtype)
    loc = int(fb.page_table[2, far])
    q = (keys[loc].float().view(kv, 1, dim) * 3).expand(kv, heads // kv, dim).reshape(1, heads, dim).expand(t, heads, dim)
    q = q.to(dtype).contiguous()
    got = O.grouped_attention(q.to(DEV), keys.to(DEV), values.to(DEV), fb, kv, 1.0, 60.0)
    pick = [0, t // 2, t - 1]
    want = plain_attention(q, keys, values, fb, kv, 1.0, 60.0, None, None, pick)
    assert err(got.cpu()[pick], want) < 2 * TOL[dtype]
    if far <= n - max(portion, 1):
        alone = values[loc].to(F).view(kv, 1, 32).expand(kv, heads // kv, 32).reshape(1, -1)
        assert err(want[-1:], alone) < 1e-2


@pytest.mark.parametrize("limit,buckets", [(30, 16), (129, 32), (700, 32), (7, 12), (100000, 8)])
def test_every_distance_gets_its_bucket(limit, buckets):
    """Equal scores, biases far apart: the weights tell every distance's bucket, in prompts and in decoding."""
    n, heads = 600, 2
    table = torch.arange(buckets)[:, None] * torch.tensor([[0.7, -0.5]])
    for dtype in TOL:
        for prefill, first in ((True, 0), (True, n - 70), (True, n - 3), (False, n - 1)):
            fb, rows = make_fb([(1, first, n - first)], DEV, prefill=prefill)
            t = n - first
            keys = torch.zeros(rows, 16, dtype=dtype)
            values = rand(rows, 24, seed=1).to(dtype)
            q = rand(t, heads, 16, seed=2).to(dtype)
            got = O.grouped_attention(q.to(DEV), keys.to(DEV), values.to(DEV), fb, 1, 1.0, 5.0, None,
                                      spread_buckets(table, limit).to(DEV))
            pick = sorted({0, t // 3, t - 1})
            want = plain_attention(q, keys, values, fb, 1, 1.0, 5.0, None, (table, limit), pick)
            assert err(got.cpu()[pick].view(-1, 24), want.view(-1, 24)) < 1.5 * TOL[dtype]


@BOTH
def test_sink_takes_its_share(dtype):
    """One key and a sink: the output is the value times e^s / (e^s + e^sink), nothing of it capped or scaled."""
    for segs, prefill in (([(1, 0, 1)], False), ([(1, 0, 80)], True)):
        fb, rows = make_fb(segs, DEV, prefill=prefill)
        t = fb.positions.shape[0]
        keys, values = torch.zeros(rows, 16, dtype=dtype), rand(rows, 16, seed=1).to(dtype)
        sink = torch.tensor([-30.0, 0.0, 1.5, 40.0])
        got = O.grouped_attention(rand(t, 4, 16).to(dtype).to(DEV), keys.to(DEV), values.to(DEV), fb, 1, 1.0, 2.0, sink.to(DEV))
        v = values[int(fb.page_table[1, 0])].to(F)
        want = v * (1.0 / (1.0 + torch.exp(sink.to(F))))[:, None]
        assert torch.allclose(got[0].view(4, 16).cpu().to(F), want, rtol=TOL[dtype], atol=1e-6)


def test_gathered_keys_and_values():
    fb, rows = make_fb([(1, 0, 70), (2, 10, 200)], DEV)
    kw, vw = 72, 136
    keys, values = rand(rows, kw, dtype=torch.bfloat16).to(DEV), rand(rows, vw, seed=1, dtype=torch.bfloat16).to(DEV)
    from minisgl.ops import native as nv
    from minisgl.ops.native import I

    reqs = torch.tensor([1, 70, 0, 0, 2, 170, 128, 40], dtype=torch.int32, device=DEV)   # slot, keys, row, first key
    total = 128 + 256
    ck, cv = torch.full((total, kw), 9.0, device=DEV).bfloat16(), torch.full((vw, total), 9.0, device=DEV).bfloat16()
    nv.call("kv_gather", nv.ptr(keys), nv.ptr(values), nv.ptr(ck), nv.ptr(cv), nv.ptr(reqs), I(2), I(total),
            nv.ptr(fb.page_table), I(fb.page_table.stride(0)), I(kw), I(vw))
    for slot, n, at, end, key0 in ((1, 70, 0, 128, 0), (2, 170, 128, 384, 40)):
        loc = fb.page_table[slot, key0:key0 + n].long()
        assert torch.equal(ck[at:at + n], keys[loc]) and torch.equal(cv[:, at:at + n], values[loc].t())
        assert float(ck[at + n:end].abs().max()) == 0 and float(cv[:, at + n:end].abs().max()) == 0


# --------------------------------------------------------------------------- short convolutions, gated delta rule
def delta_case(segs, heads, kv, d, e, taps, dtype, rate_mean=0.0, seed=0):
    fb, _ = make_fb(segs, DEV)
    t = sum(n for _, _, n in segs)
    up = lambda n: -(-n // 8) * 8
    qk, at_v = kv * d, 2 * up(kv * d)
    at_b = at_v + up(heads * e)
    c = 2 * qk + heads * e
    case = dict(fb=fb, p=rand(t, up(at_b + heads), seed=seed).to(dtype), taps=rand(taps, c, seed=seed + 1, std=0.7) + 0.3,
                before=rand(7, taps - 1, c, seed=seed + 2).to(dtype), rate=rand(t, heads * d, seed=seed + 3) + rate_mean,
                dt=rand(heads * d, seed=seed + 4), a_log=rand(heads, seed=seed + 5, std=0.5) - 1.0,
                gate=rand(t, heads * e, seed=seed + 6).to(dtype), gain=rand(e, seed=seed + 7, std=0.2) + 1.0,
                state=rand(7, heads, d, e, seed=seed + 8, std=0.3), at_b=at_b)
    for slot, start, _ in segs:           # positions below zero
        case["before"][slot, : max(taps - 1 - start, 0)] = 0
    case["cols"] = torch.cat([torch.arange(qk), up(qk) + torch.arange(qk), at_v + torch.arange(heads * e)])
    return case


def check_delta(segs, heads, kv, d, e, taps, dtype, tol, rate_mean=0.0):
    c = delta_case(segs, heads, kv, d, e, taps, dtype, rate_mean)
    fb, on = c["fb"], {k: v.to(DEV) for k, v in c.items() if isinstance(v, torch.Tensor)}
    q, k, v = O.conv_unit(on["p"], on["taps"], on["before"], fb, heads, kv, d, e)
    y = O.delta_rule(q, k, v, on["rate"], on["dt"], on["a_log"], on["p"], c["at_b"], on["gate"], on["gain"], 1e-4, on["state"],
                     on["before"], fb, heads, kv)
    row, qk = 0, kv * d
    for slot, start, n in segs:
        r = slice(row, row + n)
        x = c["p"][r].to(F)[:, c["cols"]]
        old = c["before"][slot].to(F) if start else torch.zeros(taps - 1, x.shape[1], dtype=F)
        z, keep = P.short_conv(x, c["taps"].to(F).T, old)
        qw, kw, vw = z.split([qk, qk, heads * e], 1)
        qw, kw = P.unit(qw.reshape(n, kv, d)) / math.sqrt(d), P.unit(kw.reshape(n, kv, d))
        assert err(q[r].view(n * kv, d), qw.reshape(n * kv, d)) < 2e-5 and err(k[r].view(n * kv, d), kw.reshape(n * kv, d)) < 2e-5
        assert err(v[r], vw) < TOL[dtype]
        spread = lambda s: s.repeat_interleave(heads // kv, 1)
        rate = (c["rate"][r] + c["dt"]).to(F)
        g = torch.exp(-torch.exp(c["a_log"].to(F))[:, None] * torch.nn.functional.softplus(rate).view(n, heads, d))
        beta = P.sigmoid(c["p"][r, c["at_b"]:c["at_b"] + heads].to(F))
        s0 = c["state"][slot].to(F) if start else torch.zeros(heads, d, e, dtype=F)
        o, s = P.delta_recurrence(spread(qw), spread(kw), v[r].cpu().to(F).view(n, heads, e), g, beta, s0)
        o = o / torch.sqrt((o * o).mean(-1, keepdim=True) + 1e-4) * c["gain"].to(F)
        want = o.reshape(n, heads * e) * P.sigmoid(c["gate"][r].to(F))
        assert err(y[r].reshape(n * heads, e), want.reshape(n * heads, e)) < tol, (slot, start, n)
        assert err(on["state"][slot].flatten(0, 1), s.flatten(0, 1)) < 1e-4
        if taps > 1:
            assert torch.equal(on["before"][slot].cpu(), keep.to(dtype))
        row += n


DELTA_SIZES = [(1, 1, 8, 8, 4), (4, 2, 16, 24, 3), (2, 1, 32, 64, 2), (6, 3, 20, 12, 4), (2, 2, 48, 136, 5), (3, 1, 64, 128, 1),
               (2, 2, 128, 128, 4), (2, 1, 96, 40, 4)]
DELTA_SEGS = [[(0, 0, 1), (1, 5, 1)], [(2, 0, 40)], [(3, 8, 17), (0, 0, 2), (5, 1, 1), (4, 100, 33), (1, 2, 2)]]


@BOTH
@pytest.mark.parametrize("heads,kv,d,e,taps", DELTA_SIZES + [(1, 1, 200, 72, 4), (2, 2, 130, 200, 2), (3, 3, 9, 7, 3), (2, 1, 24, 33, 4)])
@pytest.mark.parametrize("segs", DELTA_SEGS)
def test_delta_token_by_token(heads, kv, d, e, taps, segs, dtype):
    check_delta(segs, heads, kv, d, e, taps, dtype, 1.5 * TOL[dtype])


@BOTH
@pytest.mark.parametrize("heads,kv,d,e,taps", DELTA_SIZES)
@pytest.mark.parametrize("segs", [[(1, 0, 64)], [(2, 3, 200)], [(3, 8, 65), (0, 0, 2), (5, 1, 1), (4, 100, 33), (1, 0, 96)]])
def test_delta_in_chunks(heads, kv, d, e, taps, segs, dtype, monkeypatch):
    monkeypatch.setattr(C, "DELTA_CHUNKED", True)
    check_delta(segs, heads, kv, d, e, taps, dtype, max(TOL[dtype] * 1.5, 1e-4))


@pytest.mark.parametrize("rate_mean", [-12.0, -3.0, 3.0, 12.0, 60.0])
def test_delta_chunks_with_slow_and_fast_decays(rate_mean, monkeypatch):
    """A state that hardly decays over hundreds of tokens, decays on both sides of what the blocks' references allow, and
    decays that leave nothing of the token before."""
    monkeypatch.setattr(C, "DELTA_CHUNKED", True)
    check_delta([(1, 0, 300), (2, 50, 70)], 2, 1, 32, 48, 4, torch.float32, 2e-4, rate_mean)

