"""The kernels of token-pair embeddings, norms behind the sub-layers, clamped gates, element-wise recurrences, and attention in windows
(sigmoid weights, values that turn, latents with positions), one mechanism at a time, against the plain statements in
``plain_sakevik``."""
import pytest
import torch

import plain_sakevik as P
from layered_checks import rel_err as err
from layered_util import make_fb
from minisgl.models.buvalix_weight import interleave_gate
from minisgl.models.layered_config import RotaryScaling, rotary_frequencies
from minisgl.ops import api as O
from minisgl.ops import cuda_layers as CL
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


# --------------------------------------------------------------------------- embedding of token pairs
@BOTH
@pytest.mark.parametrize("d,buckets,mul", [(96, 61, (7, 13)), (50, 1009, (2654435761, 40503)), (33, 1, (3, 5)), (2048, 30, (31, 60))])
def test_pair_embedding(d, buckets, mul, dtype):
    """Tokens of portions and of decoded steps find the one before them, wherever it ran."""
    vocab = 90
    w, pairs = rand(vocab, d, dtype=torch.bfloat16), rand(buckets + 1, d, seed=1, dtype=torch.bfloat16)
    spec = {"buckets": buckets, "mul_prev": mul[0], "mul_cur": mul[1]}
    seqs = {s: torch.randint(0, vocab, (40,), generator=torch.Generator().manual_seed(s)).tolist() for s in (0, 1, 3)}
    tokens = None
    feedback = torch.zeros(7, dtype=torch.int32)
    # the second forward's segments stand in another order, and one of them is the first's neighbour in the batch
    for step, segs in enumerate([[(1, 0, 1), (0, 0, 17), (3, 0, 2)], [(3, 2, 20), (0, 17, 1), (1, 1, 16)], [(0, 18, 1), (1, 17, 1), (3, 22, 1)]]):
        decode = step == 2
        fb, rows = make_fb(segs, DEV, prefill=not decode)
        tokens = torch.full((rows,), -1, dtype=torch.int32, device=DEV) if tokens is None else tokens
        ids = torch.tensor([t for s, a, n in segs for t in seqs[s][a:a + n]], dtype=torch.int32)
        for s, a, n in segs:
            feedback[s] = seqs[s][a]
        got_ids = on(torch.zeros_like(ids) if decode else ids)
        x, act = O.embed_residual(got_ids, on(w), dtype, on(feedback) if decode else None, fb.slots, True, 1.75,
                                  positions=fb.positions, pairs=on(pairs), pair_mul=mul, tokens=tokens, fb=fb)
        want = []
        for s, a, n in segs:
            r = P.bigram_rows(seqs[s][a:a + n], seqs[s][a - 1] if a else None, spec)
            want.append(w.to(F)[seqs[s][a:a + n]] * 1.75 + pairs.to(F)[r])
        assert err(x, torch.cat(want)) < 1e-6 and err(act, torch.cat(want)) < TOL[dtype]
        assert torch.equal(got_ids.cpu(), ids) and torch.equal(tokens[fb.out_loc.long()].cpu(), ids)


# --------------------------------------------------------------------------- norms behind the sub-layers
@BOTH
@pytest.mark.parametrize("d", [96, 33, 1024, 1500, 4096, 8192, 9000])
@pytest.mark.parametrize("bias", [True, False])
def test_norm_behind_a_sub_layer(d, bias, dtype):
    t, eps = 6, 1e-3
    x, y, b, gain, last = rand(t, d), rand(t, d, seed=1, std=3.0), rand(d, seed=2, mean=1.0), rand(d, seed=3), rand(d, seed=4, mean=1.0)
    sub = (on(y), on(b) if bias else None, on(gain))
    want = x.to(F) + P.rms(y.to(F) + (b.to(F) if bias else 0.0), eps) * gain.to(F)
    normed = P.rms(want, eps) * last.to(F) * 0.3
    xd = on(x)
    rows = torch.tensor([4, 0, 4])
    got = O.residual_norm(xd, on(last), eps, dtype, 0.3, rows=on(rows), sub=sub)
    assert torch.equal(xd.cpu(), x) and got.dtype == dtype and err(got, normed[rows]) < TOL[dtype]
    got = O.residual_norm(xd, None, eps, dtype, cast=True, sub=sub)
    assert err(xd, want) < 2e-6 and err(got, want) < TOL[dtype]
    xd = on(x)
    got = O.residual_norm(xd, on(last), eps, dtype, 0.3, sub=sub)
    assert err(xd, want) < 2e-6 and err(got, normed) < TOL[dtype]
    # without a sub-layer, as before
    assert err(O.residual_norm(on(x), on(last), eps, dtype, rows=on(rows)), (P.rms(x.to(F), eps) * last.to(F))[rows]) < TOL[dtype]


# --------------------------------------------------------------------------- clamped gates
@BOTH
@pytest.mark.parametrize("limit", [0.6, 3.0])
@pytest.mark.parametrize("t,d,f", [(5, 96, 40), (130, 72, 33), (1, 20, 7), (64, 1024, 320), (3000, 128, 1100), (1, 2048, 48)])
def test_clamped_gate_projection(t, d, f, limit, dtype):
    h = rand(t, d).to(dtype)
    g, u = (rand(f, d, seed=s, std=1.5 * d ** -0.5, dtype=torch.bfloat16) for s in (1, 2))
    got = O.gated_linear(on(h), on(interleave_gate(g, u)), "clamp", limit=limit)
    x = h.to(F)
    zg, zu = x @ g.to(F).T, x @ u.to(F).T
    assert limit > 1 or (int((zg > limit).sum()) and int((zu > limit).sum()) and int((zu < -limit).sum()))
    assert got.shape == (t, -(-f // 16) * 16) and float(got[:, f:].abs().max() if f % 16 else 0) == 0
    assert err(got[:, :f], P.clamped_gate(zg, zu, limit)) < TOL[dtype]


# --------------------------------------------------------------------------- element-wise recurrence
def gru_case(width, segs, dtype, prefill=True, decay=0.0, seed=0):
    fb, _ = make_fb(segs, DEV, prefill=prefill, max_len=4096)
    t, pad = sum(n for _, _, n in segs), -width % 8
    p = rand(t, 3 * width + 2 * pad + 3, seed=seed, std=1.5)             # wider than its parts
    at_u, at_g = width + pad, 2 * (width + pad)
    bz, bu = rand(width, seed=seed + 1, mean=-decay), rand(width, seed=seed + 2, std=0.5)
    state = rand(7, width, seed=seed + 3)
    sd = on(state)
    got = O.mingru(on(p), at_u, at_g, on(bz), on(bu), sd, fb, dtype)
    want, at = [], 0
    after = state.to(F)
    pd = p.to(F)
    for slot, a, n in segs:
        rows = pd[at:at + n]
        s0 = state[slot].to(F) if a else torch.zeros(width, dtype=F)
        s, after[slot] = P.mingru_recurrence(P.sigmoid(rows[:, :width] + bz), rows[:, at_u:at_u + width] + bu, s0)
        want.append(s * P.silu(rows[:, at_g:at_g + width]))
        at += n
    assert err(got, torch.cat(want)) < TOL[dtype], segs
    assert err(sd, after) < (1e-5 if dtype == torch.float32 else 1e-4)
    untouched = [i for i in range(7) if i not in {s for s, _, _ in segs}]
    assert torch.equal(sd.cpu()[untouched], state[untouched])


@BOTH
@pytest.mark.parametrize("width", [1, 19, 64, 224, 1000, 4096])
def test_recurrence(width, dtype):
    gru_case(width, [(0, 0, 1), (3, 17, 1), (5, 0, 1)], dtype, prefill=False)
    gru_case(width, [(0, 0, 1), (3, 17, 2), (5, 5, 16)], dtype)
    gru_case(width, [(0, 0, 300), (3, 17, 1), (5, 5, 130), (1, 0, 17)], dtype, decay=2.0)


@BOTH
@pytest.mark.parametrize("ct", [8, 16, 32])
def test_parallel_recurrence_at_its_edges(ct, dtype, monkeypatch):
    """Lengths around the tiles of every form; gates that forget within a token and ones that remember all of it."""
    monkeypatch.setattr(CL, "GRU_TILES", (ct,))
    tile = 256 // ct * 8
    for n in (17, tile - 1, tile, tile + 1, 2 * tile + 9):
        gru_case(45, [(2, 7, n), (4, 0, n + 3)], dtype, decay=3.0)
    gru_case(45, [(2, 7, 2 * tile + 9)], dtype, decay=12.0)
    gru_case(45, [(2, 7, 2 * tile + 9)], dtype, decay=-12.0)


@BOTH
def test_recurrence_in_portions_carries_its_state(dtype):
    width, n = 40, 250
    p, bz, bu = on(rand(n, 3 * width, std=1.5)), on(rand(width, seed=1, mean=-3.0)), on(rand(width, seed=2))
    whole, _ = make_fb([(2, 0, n)], DEV)
    state = torch.full((7, width), float("nan"), device=DEV)
    want = O.mingru(p, width, 2 * width, bz, bu, state, whole, dtype)
    last = state[2].clone()
    state.fill_(float("nan"))
    at, out = 0, []
    for k in (2, 1, 64, 63, 3, 100, 17):
        fb, _ = make_fb([(2, at, k)], DEV, prefill=k > 1)
        out.append(O.mingru(p[at:at + k], width, 2 * width, bz, bu, state, fb, dtype))
        at += k
    assert at == n and err(torch.cat(out), want.cpu().to(F)) < TOL[dtype] and err(state[2:3], last[None].cpu().to(F)) < 1e-5


# --------------------------------------------------------------------------- norms per head, rotation, cache
@BOTH
@pytest.mark.parametrize("halves", [True, False])
@pytest.mark.parametrize("heads,kv,dim,vdim,dims", [(6, 3, 32, 24, 24), (4, 1, 16, 64, 16), (3, 3, 7, 6, 4), (16, 4, 128, 128, 64),
                                                    (2, 2, 24, 40, 0), (1, 1, 2, 2, 2), (5, 1, 12, 320, 10), (64, 8, 128, 128, 128),
                                                    (28, 4, 128, 64, 120), (96, 8, 128, 128, 64)])
@pytest.mark.parametrize("long", [0, 520])       # few tokens and many run with other blocks
def test_norm_and_rotation_per_head(heads, kv, dim, vdim, dims, long, halves, dtype):
    fb, rows = make_fb([(1, 0, 5), (2, 22, 4), (0, 900, 2)] + [(3, 30, long)] * (long > 0), DEV)
    t, n, eps, base, mul = 11 + long, (heads + kv) * dim + kv * vdim, 1e-2, 700.0, 1.3
    wide = rand(t, n + 8, std=0.3).to(dtype)          # a column slice of a wider projection
    bias, gain = rand(n, seed=1), rand(2, dim, seed=2, mean=1.0)
    freq, vfreq = rotary_frequencies(dims, base)[0] if dims else None, rotary_frequencies(vdim, base)[0]
    keys, values = (torch.zeros(rows, kv * w, dtype=dtype, device=DEV) for w in (dim, vdim))
    got, turn = O.head_store(on(wide)[:, :n], on(bias), on(gain), eps, on(freq), mul, on(vfreq), halves, keys, values, fb, heads, kv,
                             dim, vdim)
    q, k, v = (wide[:, :n].to(F) + bias.to(F)).split([heads * dim, kv * dim, kv * vdim], 1)
    pos = fb.positions.cpu()
    norm = lambda x, m, i: P.rms(x.reshape(t, m, dim), eps) * gain[i].to(F)
    rot = lambda x: P.turn(x, pos, P.frequencies({"base": base}, dims)[0], mul, halves) if dims else x
    vf = P.frequencies({"base": base}, vdim)[0]
    loc = on(fb.out_loc.cpu().long())
    limit = 2 * TOL[dtype] if dtype == torch.bfloat16 else 1e-4            # angles of 900 in 32 bits
    assert err(got.flatten(1), rot(norm(q, heads, 0)).flatten(1)) < limit
    assert err(keys[loc], rot(norm(k, kv, 1)).flatten(1)) < limit
    assert err(values[loc], P.turn(v.reshape(t, kv, vdim), pos, vf, 1.0, halves).flatten(1)) < limit
    angle = pos.to(F)[:, None] * vf
    assert float((turn.cpu().to(F) - torch.stack([torch.cos(angle), torch.sin(angle)], -1)).abs().max()) < 2e-4


# --------------------------------------------------------------------------- attention in windows
def attention_case(heads, kv, dim, vdim, window, segs, dtype, prefill=True, scale=0.4, edit=None, finish=True, seed=0, max_len=2048,
                   tol=1.0):
    fb, rows = make_fb(segs, DEV, prefill=prefill, max_len=max_len)
    t = sum(n for _, _, n in segs)
    q, keys, values = rand(t, heads, dim, seed=seed + 1), rand(rows, kv * dim, seed=seed + 2), rand(rows, kv * vdim, seed=seed + 3)
    bias = rand(heads, seed=seed + 4, mean=-1.5)
    if edit:
        edit(q, keys, values, fb)
    q, keys, values = q.to(dtype), keys.to(dtype), values.to(dtype)
    gate = rand(t, heads + 5, seed=seed + 5).to(dtype)[:, :heads] if finish else None
    pos = fb.positions.cpu()
    vf = P.frequencies({"base": 400.0}, vdim)[0]
    angle = pos.to(F)[:, None] * vf
    turn = torch.stack([torch.cos(angle), torch.sin(angle)], -1).float() if finish else None
    got = O.grouped_attention(on(q), on(keys), on(values), fb, kv, scale, window=window, wbias=on(bias), turn=on(turn),
                              gate=on(gate) if finish else None)
    want, at, table = [], 0, fb.page_table.cpu()
    for slot, a, n in segs:
        loc = table[slot, :a + n].long()
        o = P.sigmoid_attend(q[at:at + n].to(F), keys[loc].to(F).view(a + n, kv, dim), values[loc].to(F).view(a + n, kv, vdim), scale,
                             window, bias.to(F))
        if finish:
            o = P.turn(o, pos[at:at + n], vf, 1.0, True, back=True) * P.sigmoid(gate[at:at + n].to(F))[:, :, None]
        want.append(o.flatten(1))
        at += n
    want = torch.cat(want)
    assert err(got, want) < tol * TOL[dtype], (segs, window)
    return got, want


SHAPES = [(6, 3, 32, 24), (4, 1, 16, 64), (8, 2, 48, 32), (3, 3, 7, 6), (16, 4, 128, 128), (34, 1, 8, 16), (2, 1, 160, 144), (2, 2, 24, 320)]


@BOTH
@pytest.mark.parametrize("window", [1, 2, 37, 64, 128, 5000])
@pytest.mark.parametrize("shape", SHAPES)
def test_sigmoid_attention(shape, window, dtype):
    attention_case(*shape, window, [(0, 0, 1), (2, 63, 1), (1, 200, 1), (4, 36, 1)], dtype, prefill=False)
    attention_case(*shape, window, [(0, 0, 70), (2, 63, 2), (1, 130, 5), (3, 250, 1)], dtype)


@pytest.mark.parametrize("form", ["flash", "rows"])
@pytest.mark.parametrize("window", [1, 50, 64, 129, 300, 5000])
@pytest.mark.parametrize("shape", [(6, 3, 32, 32), (4, 2, 128, 128), (2, 1, 64, 96), (3, 1, 72, 64)])
@pytest.mark.parametrize("finish", [True, False])
def test_both_kernels_of_prompts(shape, window, form, finish, monkeypatch):
    monkeypatch.setattr(C, "GROUPED_PREFILL", form)
    segs = [(0, 0, 300), (2, 190, 140), (1, 700, 2), (3, 5, 64)]
    attention_case(*shape, window, segs, torch.bfloat16, finish=finish, tol=1.3)


def test_prompts_without_whole_vector_turns_use_the_row_kernel():
    attention_case(4, 2, 32, 40, 90, [(0, 0, 200), (1, 64, 130)], torch.bfloat16)


@BOTH
@pytest.mark.parametrize("form", ["flash", "rows", "decode"])
@pytest.mark.parametrize("window", [1, 33, 64, 127, 128, 200])
def test_one_loud_key_at_the_edge_of_the_window(form, window, dtype, monkeypatch):
    """Everything else weighs next to nothing: the key at distance window - 1 decides the row, the one at distance window must not."""
    if form == "flash" and dtype == torch.float32:
        pytest.skip("the prompt kernel takes bf16")
    monkeypatch.setattr(C, "GROUPED_PREFILL", form if form != "decode" else "auto")
    heads, dim = 2, 32
    row = 260
    for inside in (True, False):
        at = row - window + (1 if inside else 0)

        def edit(q, keys, values, fb):
            q.zero_()
            keys.zero_()
            q[:, :, 0] = -20.0               # every key but the loud one: sigmoid(-20 * 0.4 ...)
            keys[:, 0] = 2.0
            loc = int(fb.page_table[1, at])
            keys[loc, 0] = -2.0
            values[loc] *= 3.0

        if form == "decode":
            segs = [(0, 3, 1), (1, row, 1)]
        else:
            segs = [(0, 0, 3), (1, 100, row + 1 - 100)]
        got, want = attention_case(heads, 1, dim, 32, window, segs, dtype, prefill=form != "decode", scale=0.4, edit=edit, finish=False,
                                   tol=2.0)
        assert (float(want[-1].abs().max()) > 0.1) == inside


def test_weights_are_not_normalised():
    """Ten equal keys weigh ten times as much as one."""
    fb, rows = make_fb([(0, 9, 1)], DEV, prefill=False)
    for dtype in (torch.bfloat16, torch.float32):
        q, keys, values = (torch.ones(1, 1, 16), torch.ones(rows, 16), torch.ones(rows, 16))
        for window, n in ((1, 1), (10, 10)):
            got = O.grouped_attention(on(q.to(dtype)), on(keys.to(dtype)), on(values.to(dtype)), fb, 1, 0.0, window=window,
                                      wbias=torch.zeros(1, device=DEV))
            assert float((got.float() - 0.5 * n).abs().max()) < 1e-3


@BOTH
def test_softmax_in_a_window(dtype):
    """The window beside a softmax, in every kernel."""
    heads, kv, dim, vdim = 4, 2, 32, 32
    for window in (1, 60, 128):
        for segs, prefill in (([(0, 0, 200), (2, 63, 3)], True), ([(0, 100, 1), (2, 3, 1)], False)):
            fb, rows = make_fb(segs, DEV, prefill=prefill)
            t = sum(n for _, _, n in segs)
            q, keys, values = rand(t, heads, dim).to(dtype), rand(rows, kv * dim, seed=1).to(dtype), rand(rows, kv * vdim, seed=2).to(dtype)
            got = O.grouped_attention(on(q), on(keys), on(values), fb, kv, 0.3, window=window)
            want, at = [], 0
            for slot, a, n in segs:
                loc = fb.page_table.cpu()[slot, :a + n].long()
                wide = lambda x, w: x[loc].to(F).view(a + n, kv, w).repeat_interleave(2, 1)
                want.append(P.softmax_attend(q[at:at + n].to(F), wide(keys, dim), wide(values, vdim), 0.3, window).flatten(1))
                at += n
            assert err(got, torch.cat(want)) < 1.3 * TOL[dtype], (window, segs)


# --------------------------------------------------------------------------- latent attention with positions, in windows
@BOTH
@pytest.mark.parametrize("heads,dim,rot,rank,scaling", [(4, 24, 16, 48, (4.0, 64, 8.0, 1.0)), (3, 7, 6, 11, None), (1, 1, 2, 1, None),
                                                        (16, 96, 32, 512, (8.0, 4096, 32.0, 1.0))])
def test_latent_rows_and_queries_turn(heads, dim, rot, rank, scaling, dtype):
    fb, rows = make_fb([(1, 0, 5), (2, 22, 4), (0, 900, 2)], DEV)
    t, eps, base, up = 11, 1e-2, 3000.0, lambda n: -(-n // 8) * 8
    at_rot = up(heads * dim)
    at_c = at_rot + up(heads * rot)
    p, gain = rand(t, at_c + up(rank + rot)).to(dtype), rand(rank, seed=1, mean=1.0)
    freq, mul = rotary_frequencies(rot, base, RotaryScaling(*scaling) if scaling else None)
    want_f, want_mul = P.frequencies({"base": base, "scaling": dict(zip(("factor", "original", "fast", "slow"), scaling)) if scaling else None}, rot)
    pos, pf = fb.positions.cpu(), p.to(F)
    q = P.turn(pf[:, at_rot:at_rot + heads * rot].view(t, heads, rot), pos, want_f, want_mul, False)
    c = P.rms(pf[:, at_c:at_c + rank], eps) * gain.to(F)
    r = P.turn(pf[:, None, at_c + rank:at_c + rank + rot], pos, want_f, want_mul, False)[:, 0]
    limit = TOL[dtype] if dtype == torch.bfloat16 else 1e-4
    for whole in (False, True):
        cache, pd = torch.zeros(rows, rank + rot, dtype=dtype, device=DEV), on(p)
        got = O.latent_rotate_store(pd, at_rot, at_c, on(gain), eps, on(freq), mul, cache, fb, heads, dim, whole)
        assert err(cache[on(fb.out_loc.cpu().long())], torch.cat([c, r], 1)) < limit
        if whole:
            want = torch.cat([pf[:, :heads * dim].view(t, heads, dim), q], -1).flatten(1)
            assert torch.equal(pd.cpu(), p) and err(got, want) < limit
        else:
            assert got is None and err(pd[:, at_rot:at_rot + heads * rot], q.flatten(1)) < limit
            assert torch.equal(pd[:, :at_rot].cpu(), p[:, :at_rot]) and torch.equal(pd[:, at_c:].cpu(), p[:, at_c:])


def latent_want(q, q_rot, cache, fb, segs, rank, scale, window):
    """q [T, H, rank], q_rot [T, H, rot] over the cached rows, which are keys and (their first part) values alike."""
    out, at, table = [], 0, fb.page_table.cpu()
    for slot, a, n in segs:
        rows = cache[table[slot, :a + n].long()].to(F)
        k = rows[:, None].expand(-1, q.shape[1], -1)
        whole = torch.cat([q[at:at + n].to(F), q_rot[at:at + n].to(F)], -1)
        out.append(P.softmax_attend(whole, k, k[..., :rank], scale, window))
        at += n
    return torch.cat(out)


@BOTH
@pytest.mark.parametrize("window", [1, 50, 64, 129, 5000])
@pytest.mark.parametrize("heads,rank,rot", [(4, 48, 16), (16, 128, 64), (3, 11, 6), (1, 1, 2), (20, 192, 64), (5, 512, 64), (8, 576, 64), (2, 320, 32)])
def test_latent_attention(heads, rank, rot, window, dtype):
    for segs, prefill in (([(0, 0, 1), (2, 63, 1), (1, 200, 1)], False), ([(0, 0, 70), (2, 63, 2), (1, 130, 5), (3, 250, 1)], True)):
        fb, rows = make_fb(segs, DEV, prefill=prefill)
        t, scale = sum(n for _, _, n in segs), 0.7 * (rank + rot) ** -0.5
        q, cache = rand(t, heads, rank, seed=1).to(dtype), rand(rows, rank + rot, seed=2).to(dtype)
        wide = rand(t, 8 + heads * rot + 8, seed=3).to(dtype)
        wide = wide[:, : wide.shape[1] // 8 * 8].contiguous() if rot % 8 == 0 else wide
        got = O.latent_attention(on(q), on(cache), fb, scale, on(wide)[:, 8:8 + heads * rot], window)
        want = latent_want(q, wide[:, 8:8 + heads * rot].reshape(t, heads, rot), cache, fb, segs, rank, scale, window)
        assert err(got.flatten(1), want.flatten(1)) < 1.3 * TOL[dtype], (segs, window)


@pytest.mark.parametrize("window", [1, 50, 64, 129, 300, 5000])
@pytest.mark.parametrize("heads,dim,rot,vdim,rank", [(4, 24, 16, 40, 48), (2, 96, 32, 128, 256), (3, 64, 64, 64, 72)])
def test_expanded_latents(heads, dim, rot, vdim, rank, window):
    segs = [(0, 0, 300), (2, 190, 140), (1, 700, 2), (3, 5, 64)]
    fb, rows = make_fb(segs, DEV)
    t, scale = sum(n for _, _, n in segs), (dim + rot) ** -0.5
    bf = torch.bfloat16
    q, cache = rand(t, heads * (dim + rot), seed=1).to(bf), rand(rows, rank + rot, seed=2).to(bf)
    uk, uv = rand(heads, dim, rank, seed=3, std=rank ** -0.5).to(bf), rand(heads * vdim, rank, seed=4, std=rank ** -0.5).to(bf)
    whole = torch.zeros(heads, dim + rot, rank + rot, dtype=bf)
    whole[:, :dim, :rank], whole[:, dim:, rank:] = uk, torch.eye(rot)
    got = O.expanded_attention(on(q), on(cache), fb, on(whole.view(-1, rank + rot)), on(uv), heads, scale, window)
    want, at, table = [], 0, fb.page_table.cpu()
    for slot, a, n in segs:
        c = cache[table[slot, :a + n].long()].to(F)
        k = torch.cat([torch.einsum("jr,hdr->jhd", c[:, :rank], uk.to(F)), c[:, None, rank:].expand(-1, heads, -1)], -1)
        v = (c[:, :rank] @ uv.to(F).T).view(a + n, heads, vdim)
        want.append(P.softmax_attend(q[at:at + n].to(F).view(n, heads, -1), k, v, scale, window).flatten(1))
        at += n
    assert err(got, torch.cat(want)) < 1.5 * TOL[bf]


@BOTH
@pytest.mark.parametrize("window", [1, 33, 64, 127, 128, 200])
@pytest.mark.parametrize("prefill", [True, False])
def test_one_loud_latent_at_the_edge_of_the_window(window, prefill, dtype):
    """A score that stands out, by the turned part alone: just inside it takes the whole row, just outside nothing."""
    heads, rank, rot, row = 2, 32, 16, 260
    segs = [(0, 0, 3), (1, 100, row + 1 - 100)] if prefill else [(0, 3, 1), (1, row, 1)]
    fb, rows = make_fb(segs, DEV, prefill=prefill)
    t = sum(n for _, _, n in segs)
    for inside in (True, False):
        at = row - window + (1 if inside else 0)
        cache = rand(rows, rank + rot, seed=2)
        cache[:, rank:] = 0.0
        loud = int(fb.page_table[1, at])
        cache[loud, rank] = 10.0
        cache[loud, :rank] += 5.0
        q, q_rot = rand(t, heads, rank, seed=1, std=0.1), torch.zeros(t, heads * rot)
        q_rot[:, ::rot] = 3.0
        q, q_rot, cache = q.to(dtype), q_rot.to(dtype), cache.to(dtype)
        got = O.latent_attention(on(q), on(cache), fb, 1.0, on(q_rot), window)
        want = latent_want(q, q_rot.view(t, heads, rot), cache, fb, segs, rank, 1.0, window)
        assert err(got.flatten(1), want.flatten(1)) < 1.3 * TOL[dtype]
        assert (float(want[-1].mean()) > 3.0) == inside
