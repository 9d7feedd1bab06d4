"""Operator facade used by the model.

Each function has two bodies: CUDA tensors go to the hand-written sm_100a kernels (``ops/cuda.py`` ->
``libdsv4_b200.so``), CPU tensors to the PyTorch oracle in ``ops/ref.py``.  There is no third path: a CUDA
tensor never falls back to PyTorch silently (``cuda.py`` raises when the library is missing).
"""
from __future__ import annotations

import torch

from . import gemm as _gemm
from . import ref

gemm_bf16 = _gemm.gemm_bf16
gemm_fp8 = _gemm.gemm_fp8
gemm_bf16_grouped = _gemm.gemm_bf16_grouped
linear = _gemm.linear
grouped_linear = _gemm.grouped_linear


def _cu():
    from . import cuda

    return cuda


# --------------------------------------------------------------------------- page-table helpers (CPU path)
def _locs(fb, pos):
    """Token locations of (row slot, position) pairs; pos [T,n] may be negative (-> -1)."""
    p = pos.clamp_min(0).long()
    loc = fb.page_table[fb.slots.long()[:, None], p]
    return torch.where(pos >= 0, loc, torch.full_like(loc, -1))


def swa_rows(fb, swa_map, ps: int, window: int):
    off = torch.arange(window - 1, -1, -1, device=fb.positions.device)
    pos = fb.positions.long()[:, None] - off[None, :]
    loc = _locs(fb, pos).long()
    slot = swa_map[(loc.clamp_min(0) // ps)].long()
    row = slot * ps + loc.clamp_min(0) % ps
    return torch.where((loc >= 0) & (slot >= 0), row, torch.full_like(row, -1))


def comp_rows_all(fb, ps: int, ratio: int, width: int):
    j = torch.arange(width, device=fb.positions.device)[None, :]
    n = ((fb.positions.long() + 1) // ratio)[:, None]
    loc = _locs(fb, torch.where(j < n, j * ratio + ratio - 1, torch.full_like(j, -1))).long()
    return torch.where(loc >= 0, ref.comp_row(loc.clamp_min(0), ps, ratio), torch.full_like(loc, -1))


def comp_rows_from_idx(fb, idx, ps: int, ratio: int):
    loc = _locs(fb, torch.where(idx >= 0, idx.long() * ratio + ratio - 1, torch.full_like(idx.long(), -1))).long()
    return torch.where(loc >= 0, ref.comp_row(loc.clamp_min(0), ps, ratio), torch.full_like(loc, -1))


# --------------------------------------------------------------------------- index audit (MINISGL_DEBUG_BOUNDS=1)
INDEX_TAGS = {"input_ids": 1, "positions": 2, "slots": 3, "out_loc": 4, "page_table": 5, "expert_ids": 6,
              "indexer_topk": 7}


def check_index(idx, lo: int, hi: int, what: str) -> None:
    """Every entry of ``idx`` must lie in [lo, hi).  CUDA: a device kernel records a violation in the status word
    (no synchronisation; ``native.assert_device_ok()`` raises it); CPU: raises at once."""
    if idx.is_cuda:
        return _cu().check_index(idx.contiguous(), lo, hi, INDEX_TAGS[what])
    if idx.numel() and (int(idx.min()) < lo or int(idx.max()) >= hi):
        raise IndexError(f"{what}: index outside [{lo}, {hi})")


# --------------------------------------------------------------------------- elementwise
def embed(ids, weight, m: int, feedback=None, slots=None):
    """feedback [slots+1] int32 / slots [T]: row t embeds the token ``feedback[slots[t]]`` (the previous step's sample,
    kept on the device) and stores it into ``ids[t]``."""
    if ids.is_cuda:
        return _cu().embed(ids, weight, m, feedback, slots)
    if feedback is not None:
        ids.copy_(feedback[slots.long()])
    return weight[ids.long()].unsqueeze(1).repeat(1, m, 1)


def greedy_tokens(logits, v_base: int, slots, num_valid, token_feedback, out=None, comm_ctx=None):
    """Greedy sample of every row (lowest index wins ties) into ``out`` [rows] int32 and, for valid rows, into
    ``token_feedback[slots[row]]``.  ``logits`` may be one rank's vocabulary shard (first column = token v_base)."""
    if logits.is_cuda:
        return _cu().greedy_tokens(logits, v_base, slots, num_valid, token_feedback, out, comm_ctx)
    tok = (logits.float().argmax(-1) + v_base).to(torch.int32)
    if out is None:
        out = torch.empty_like(tok)
    out.copy_(tok)
    n = logits.shape[0] if num_valid is None else int(num_valid)
    token_feedback[slots[:n].long()] = tok[:n]
    return out


def rms_norm(x, weight, eps: float, want_q: bool = False):
    """want_q: returns (out, (e4m3, scales)) -- on CUDA the normalising kernel writes the quantisation too."""
    if x.is_cuda:
        return _cu().rms_norm(x, weight, eps, want_q)
    out = ref.rms_norm(x, weight, eps)
    return (out, fp8_quant(out)) if want_q else out


def fp8_quant(x, block: int = 128):
    if x.is_cuda:
        return _cu().fp8_quant(x, block)
    from . import quant

    return quant.fp8_act_quant(x.contiguous(), block)


def silu_mul_clamp(gate_up, limit):
    if gate_up.is_cuda:
        return _cu().silu_mul_clamp(gate_up, limit)
    return ref.silu_mul_clamp(gate_up, limit)


def silu_mul_clamp_quant(gate_up, limit):
    """(e4m3, scales) of the SwiGLU activation (one kernel on CUDA)."""
    if gate_up.is_cuda:
        return _cu().silu_mul_clamp_quant(gate_up, limit)
    return fp8_quant(ref.silu_mul_clamp(gate_up, limit))


def add_cast(routed, shared, num_valid=None):
    if routed.is_cuda:
        return _cu().add_cast(routed, shared, num_valid)
    out = (routed.float() + shared.float()).to(routed.dtype)
    if num_valid is not None:
        out[int(num_valid):] = 0
    return out


def rope_tail(x, positions, spec, inverse: bool = False):
    if x.is_cuda:
        return _cu().rope_tail(x, positions, spec, inverse)
    return ref.rope_tail(x, positions, spec, inverse).to(x.dtype)


def q_kv_norm_rope_store(q, kv, positions, kv_w, eps, spec, swa_cache, out_loc, swa_map, ps: int, qat: bool):
    if q.is_cuda:
        return _cu().q_kv_norm_rope_store(q, kv, positions, kv_w, eps, spec, swa_cache, out_loc, swa_map, ps, qat)
    qo, ko = ref.q_kv_norm_rope(q, kv, positions, kv_w, eps, spec, qat)
    loc = out_loc.long()
    slot = swa_map[loc.clamp_min(0) // ps].long()
    ok = (loc >= 0) & (slot >= 0)
    swa_cache[(slot * ps + loc % ps)[ok]] = ko[ok]
    return qo, ko


# --------------------------------------------------------------------------- hyper-connections
def hc_pre(x, fn, scale, base, iters, eps, norm_eps, norm_w=None, want_q: bool = False, out=None):
    """Returns (y, post, comb); with ``norm_w`` y is additionally RMS-normalised (fused on CUDA); with ``want_q``
    a fourth item, the (e4m3, scales) quantisation of y (also fused on CUDA).  ``out`` (CUDA only): result rows
    (y, q, s) to write into."""
    if x.is_cuda:
        return _cu().hc_pre(x, fn, scale, base, iters, eps, norm_eps, norm_w, want_q, out)
    y, post, comb = ref.hc_pre(x, fn, scale, base, iters, eps, norm_eps)
    if norm_w is not None:
        y = ref.rms_norm(y, norm_w, norm_eps)
    return (y, post, comb, fp8_quant(y)) if want_q else (y, post, comb)


def hc_post(y, residual, post, comb):
    if y.is_cuda:
        return _cu().hc_post(y, residual, post, comb)
    return ref.hc_post(y, residual, post, comb)


def hc_head(x, fn, scale, base, eps, norm_eps, norm_w=None):
    if x.is_cuda:
        return _cu().hc_head(x, fn, scale, base, eps, norm_eps, norm_w)
    y = ref.hc_head(x, fn, scale, base, eps, norm_eps)
    return ref.rms_norm(y, norm_w, norm_eps) if norm_w is not None else y


# --------------------------------------------------------------------------- compressors
def compress(proj, fb, ratio: int, d: int, ape, ring, ckpt, ps: int):
    """Pools group boundaries of this call and then carries the call's rows into the ring / checkpoint state."""
    if proj.is_cuda:
        return _cu().compress(proj, fb, ratio, d, ape, ring, ckpt, ps)
    pooled = ref.compress_pool(proj, fb.positions, fb.slots, ratio, d, ape, ring, ckpt, fb.page_table, ps)
    ref.compress_state_store(proj, fb.positions, fb.slots, ratio, d, ape, ring, ckpt, fb.page_table, ps)
    return pooled


def compress_store(pooled, fb, norm_w, eps, spec, cache, ps: int, ratio: int):
    if pooled.is_cuda:
        return _cu().compress_store(pooled, fb, norm_w, eps, spec, cache, ps, ratio)
    ok = ((fb.positions.long() + 1) % ratio == 0) & (fb.out_loc >= 0)
    if bool(ok.any()):
        y = ref.compress_norm_rope(pooled[ok], fb.positions[ok].long(), norm_w, eps, spec, ratio)
        cache[ref.comp_row(fb.out_loc[ok].long(), ps, ratio)] = y


def indexer_q_encode(q, weights, positions, spec, softmax_scale, head_scale):
    if q.is_cuda:
        return _cu().indexer_q_encode(q, weights, positions, spec, softmax_scale, head_scale)
    return ref.indexer_q_encode(q, weights, positions, spec, softmax_scale, head_scale)


def indexer_kv_store(pooled, fb, norm_w, eps, spec, vals, scales, ps: int):
    if pooled.is_cuda:
        return _cu().indexer_kv_store(pooled, fb, norm_w, eps, spec, vals, scales, ps)
    ok = ((fb.positions.long() + 1) % 4 == 0) & (fb.out_loc >= 0)
    if bool(ok.any()):
        codes, sc = ref.indexer_kv_encode(pooled[ok], fb.positions[ok].long(), norm_w, eps, spec)
        rows = ref.comp_row(fb.out_loc[ok].long(), ps, 4)
        vals[rows] = codes
        scales[rows] = sc


def indexer_select(qc, wf, vals, scales, fb, ps: int, k: int):
    """Top-k compressed entries per token: (idx int32 [T,k] of compressed indices j, -1 padded; len int32 [T])."""
    if qc.is_cuda:
        return _cu().indexer_select(qc, wf, vals, scales, fb, ps, k)
    width = max(fb.max_context // 4, 1)
    rows = comp_rows_all(fb, ps, 4, width)
    lens = ((fb.positions.long() + 1) // 4).to(torch.int32)
    logits = ref.indexer_logits(qc, wf, vals, scales, rows, lens)
    return ref.topk_select(logits, lens, k)


# --------------------------------------------------------------------------- attention
def attention(q, fb, swa_cache, swa_map, comp_cache, ratio: int, topk_idx, topk_len, sink, scale, ps: int,
              window: int, out_rope=None):
    """``out_rope``: also rotate the last ``rotary_dim`` dims of every output row by minus its position (fused into
    the kernel's epilogue on CUDA, :func:`rope_tail` with ``inverse=True`` on the oracle path)."""
    if q.is_cuda:
        return _cu().attention(q, fb, swa_cache, swa_map, comp_cache, ratio, topk_idx, topk_len, sink, scale, ps,
                               window, out_rope)
    srows = swa_rows(fb, swa_map, ps, window)
    crows = None
    if ratio == 4:
        idx = torch.where((topk_len > 0)[:, None], topk_idx, torch.full_like(topk_idx, -1))
        crows = comp_rows_from_idx(fb, idx, ps, 4)
    elif ratio:
        crows = comp_rows_all(fb, ps, ratio, max(fb.max_context // ratio, 1))
    o = ref.sparse_attention(q, comp_cache, crows, swa_cache, srows, sink, scale)
    return rope_tail(o, fb.positions, out_rope, inverse=True) if out_rope is not None else o


# --------------------------------------------------------------------------- MoE
def moe_gate(y, gate_w, bias, topk, scaling, scoring, tid2eid, token_ids, num_valid=None, gate=None):
    if y.is_cuda:
        return _cu().moe_gate(y, gate_w, bias, topk, scaling, scoring, tid2eid, token_ids, num_valid, gate)
    idx, w = ref.moe_gate(y, gate_w, bias, topk, scaling, scoring, tid2eid, token_ids)
    if num_valid is not None:
        idx[int(num_valid):] = -1
        w[int(num_valid):] = 0
    return idx, w


def moe_experts(y, idx, w, w13, s13, w2, s2, limit, expert_base: int = 0):
    if y.is_cuda:
        return _cu().moe_experts(y, idx, w, w13, s13, w2, s2, limit, expert_base)
    e_local = w13.shape[0]
    local = idx - expert_base
    local = torch.where((local >= 0) & (local < e_local) & (idx >= 0), local, torch.full_like(local, -1))
    return ref.moe_experts(y, local, w, w13, s13, w2, s2, limit)


# --------------------------------------------------------------------------- fp32 residual stream, experts in bf16
def _layers(t):
    """The bodies of the operators below: kernels for CUDA tensors, plain PyTorch for CPU tensors."""
    from . import cuda_layers, ref_layers

    return cuda_layers if t.is_cuda else ref_layers


def embed_residual(ids, weight, dtype, feedback=None, slots=None, want_act: bool = False, mul: float = 1.0, table=None,
                   positions=None, streams=None, pairs=None, pair_mul=(0, 0), tokens=None, fb=None):
    """(x = embedding * mul + table[position] fp32 [T, D], the same rows as activations of ``dtype`` or None); feedback / slots
    as in :func:`embed`.  ``table``: learned position vectors or None.  ``streams``: x is that many copies [T, streams, D].
    ``pairs`` [n + 1, D]: row (token before * pair_mul[0] + token * pair_mul[1]) mod n is added, row n at position 0; ``tokens`` [token
    locations] int32 keeps the sequences' tokens between forwards (needs slots, positions and ``fb``)."""
    return _layers(ids).embed_residual(ids, weight, dtype, feedback, slots, want_act, mul, table, positions, streams, pairs,
                                       pair_mul, tokens, fb)


def stream_norm(x, eps: float, dtype, pre=None, post=None, sub=None, experts=None, rows=None, keep: bool = True):
    """One step of fp32 residual streams x [T, S, D] with constant mixing weights.  With ``post`` = out [S] | mix [S, S] (from,
    to), flat: x_t <- sum_s mix[s, t] x_s + out[t] y for y = ``sub`` [T, D] fp32 + the weighted rows of ``experts`` = (expert rows
    [T*k, D], weights [T, k], ids [T, k], n, h [T, D]); ids from n on stand for h itself, negative ones for nothing.  With ``pre``
    = in [S] | gain: returns u / rms(u) * gain as activations for u = sum_s in[s] x_s, else None.  ``rows``: only these are
    computed and returned.  keep=False (always with ``rows``): x itself may be left as it was."""
    return _layers(x).stream_norm(x, eps, dtype, pre, post, sub, experts, rows, keep and rows is None)


def residual_norm(x, gain, eps: float, dtype, mul: float = 1.0, rows=None, add=None, add2=None, vec=None, experts=None,
                  cast: bool = False, sub=None):
    """Adds whatever is given to the fp32 stream x (in place): ``sub`` = (y [T, D] fp32, bias [D] or None, gain): (y + bias) /
    rms(y + bias) * gain; ``add`` / ``add2`` [T, D] fp32, ``vec`` [D] fp32, ``experts`` = (expert rows [T*k, D], weights [T, k], ids
    [T, k]).  Then returns x / rms(x) * gain * mul as activations; with gain None nothing is normed and the sum itself is returned if
    ``cast`` is set.  ``rows``: the rows wanted (only ``sub`` is added then, and x itself is left as it was)."""
    return _layers(x).residual_norm(x, gain, eps, dtype, mul, rows, add, add2, vec, experts, cast, sub)


def route_topk(h, weight, bias, top: int, num_valid=None, kind: str = "selected", scale: float = 1.0):
    """Router of a mixture, logits z = h W^T in fp32; the weights are times ``scale``.  kind "selected": the ``top`` largest
    z + b (lower id on ties) and the softmax over them; "softmax": p = softmax(z) over all, the ``top`` largest p + b, weighted
    with their p.  Rows >= num_valid get id -1."""
    return _layers(h).route_topk(h, weight, bias, top, num_valid, kind, scale)


def gated_experts(h, idx, wts, w13, w2):
    """silu(gate) * up experts: w13 [E, 2, F, D] (gate, up), w2 [E, D, F], bf16.  Returns the chosen experts' outputs
    [T*k, D], not weighted yet (``residual_norm`` adds them up)."""
    return _layers(h).gated_experts(h, idx, wts, w13, w2)


# --------------------------------------------------------------------------- latent attention, recurrent mixing
def latent_store(x, gain, eps: float, cache, fb):
    """cache[out_loc[t]] = x[t] / rms(x[t]) * gain (x may be a column slice)."""
    return _layers(x).latent_store(x, gain, eps, cache, fb)


def latent_rotate_store(p, at_rot: int, at_c: int, gain, eps: float, freq, mul: float, cache, fb, heads: int, dim: int,
                        whole: bool = False):
    """Behind the projection of latent attention with positions, p [T, ..]: the heads' unrotated parts [H * dim] from column 0, the
    parts that turn [H * rot] from ``at_rot``, latent [R] | shared part that turns [rot] from ``at_c``.  Neighbouring values turn by
    position * freq (rot / 2 frequencies), cos and sin times ``mul``.  cache[out_loc[t]] = [latent / rms * gain | turned part].  The
    queries' parts turn in place; with ``whole`` they come out behind the unrotated ones instead, [T, H * (dim + rot)]."""
    return _layers(p).latent_rotate_store(p, at_rot, at_c, gain, eps, freq, mul, cache, fb, heads, dim, whole)


def latent_attention(q, cache, fb, scale: float, q_rot=None, window: int = 0):
    """Causal attention of every (token, head) row over its request's cached latents, which are keys and values alike:
    q [T, H, R] (key up-projection absorbed) -> [T, H, R].  ``q_rot`` [T, H * rot] (may be a column slice): the score also has the
    product with the last rot values of a cache row.  ``window`` > 0: position i sees the keys i - window + 1 .. i."""
    return _layers(q).latent_attention(q, cache, fb, scale, q_rot, window)


def prefers_expanded(q, fb, heads: int, dim: int, vdim: int, rank: int, rot: int = 0, window: int = 0) -> bool:
    """Whether :func:`expanded_attention` is the cheaper form for this forward (long prompt portions)."""
    return _layers(q).prefers_expanded(q.dtype, fb, heads, dim, vdim, rank, rot, window)


def expanded_attention(q, cache, fb, uk, uv, heads: int, scale: float, window: int = 0):
    """The same attention with keys W_uk c and values W_uv c expanded from the requests' cached rows c (values: from the first R
    columns): q [T, H*dim] (a column slice), uk [H*dim, width], uv [H*vdim, R] -> [T, H*vdim]."""
    return _layers(q).expanded_attention(q, cache, fb, uk, uv, heads, scale, window)


def mingru(p, at_u: int, at_g: int, bias_z, bias_u, state, fb, dtype):
    """Element-wise gated recurrence, S <- (1 - z) S + z c with z = sigmoid(p_z + bias_z), u = p_u + bias_u, c = u + 1/2 for u >= 0,
    else sigmoid(u); p fp32 [T, ..]: z from column 0, u from ``at_u``, g from ``at_g``; S [width] fp32 in ``state`` [slots + 1, width].
    Returns S * silu(p_g) as activations [T, width]."""
    return _layers(p).mingru(p, at_u, at_g, bias_z, bias_u, state, fb, dtype)


def shift_mix(x, gain, eps: float, mu, prev, tail, fb, dtype):
    """Norm and token shift: h = x / rms(x) * gain, h' = the previous token's h; returns [T, n*D], mix m being
    h + (h' - h) mu[m].  prev [slots+1, D]: every slot's last h, read by the first row of a portion.  tail: scratch of
    the same shape (``wkv`` moves a portion's last row from there to prev)."""
    return _layers(x).shift_mix(x, gain, eps, mu, prev, tail, fb, dtype)


def wkv(p, a, w0, u, gain, state, prev, tail, fb, heads: int, eps: float):
    """Recurrence with decay exp(-exp(a + w0)), bonus u, per-head norm, gain and silu gate (csrc/wkv.cu).  p [T, 4*H*d]:
    r | k | v | g; a fp32 [T, H*d]; state fp32 [slots+1, H, d, d] is advanced.  Returns [T, H*d]."""
    return _layers(p).wkv(p, a, w0, u, gain, state, prev, tail, fb, heads, eps)


# --------------------------------------------------------------------------- layer norms, grouped attention, delta rule
def _mixers(t):
    from . import cuda_mixers, ref_mixers

    return cuda_mixers if t.is_cuda else ref_mixers


def residual_layer_norm(x, eps: float, dtype, norm=None, sub=None, add=None, rows=None, keep: bool = True):
    """One step of the fp32 stream x [T, D] with layer norms around the sub-layers: x += N(y; w, b) for ``sub`` = (y fp32
    [T, D], w, b), then x += ``add`` [T, D] (activations), then returns N(x; w, b) as activations for ``norm`` = (w, b), else
    None.  ``rows``: only these rows are computed and returned.  keep=False (always with ``rows``): x itself may be left
    as it was."""
    return _mixers(x).residual_layer_norm(x, eps, dtype, norm, sub, add, rows, keep and rows is None)


def gated_linear(h, w, act: str, block: int = 16, limit: float = 0.0):
    """act(gate h) * (up h), act "gelu_tanh" or "silu", for w [2F, D] in alternating blocks of ``block`` gate and up rows -> [T, F].
    act "clamp": g sigmoid(1.702 g) (u + 1) for g = min(gate h, limit), u = up h clamped to [-limit, limit]."""
    return _mixers(h).gated_linear(h, w, act, block, limit)


def rotate_store(qkv, bias, freq, q_temp, keys, values, fb, heads: int, kv_heads: int, dim: int, vdim: int, gain=None,
                 unit_v: bool = False, eps: float = 0.0, v_mul: float = 1.0):
    """Behind the projection q | k | v of grouped attention: adds ``bias`` (or None); with ``gain`` divides q and k by the root
    mean square of all their rows and multiplies by it; with ``unit_v`` divides every head's values by their root mean square;
    multiplies the values by ``v_mul``; turns neighbouring pairs of the first
    2 * len(freq) dimensions of every q and k head by position * freq (or not), multiplies q by its temperature
    1 + coef * ln(floor((position + 1) / every) + 1) for q_temp = (coef, every), writes keys and values to the rows
    ``fb.out_loc`` of the caches and returns q [T, H, dim]."""
    return _mixers(qkv).rotate_store(qkv, bias, freq, q_temp, keys, values, fb, heads, kv_heads, dim, vdim, gain, unit_v, eps,
                                     v_mul)


def head_store(qkv, bias, gain, eps: float, freq, mul: float, vfreq, halves: bool, keys, values, fb, heads: int, kv_heads: int,
               dim: int, vdim: int):
    """Behind the projection q | k | v of grouped attention: adds ``bias`` (or None); with ``gain`` [2, dim] divides every q and k head
    by its root mean square and multiplies by its row; turns the first 2 * len(freq) dimensions of q and k heads by position * freq, cos
    and sin times ``mul``; with ``vfreq`` [vdim / 2] turns whole value heads.  Partners are dimensions i and i + half of the turned
    ones (``halves``), or neighbours.  Writes keys and values to the rows ``fb.out_loc`` of the caches.  Returns (q [T, H, dim], cos
    and sin of the values' angles fp32 [T, vdim / 2, 2] or None)."""
    return _mixers(qkv).head_store(qkv, bias, gain, eps, freq, mul, vfreq, halves, keys, values, fb, heads, kv_heads, dim, vdim)


def grouped_attention(q, keys, values, fb, kv_heads: int, scale: float, softcap: float = 0.0, sink=None, rel=None, slope=None,
                      chunk: int = 0, window: int = 0, wbias=None, turn=None, gate=None):
    """Causal attention of q [T, H, dim] over the cached keys and values of every request, H / kv_heads query heads to a key
    head.  score = softcap * tanh(q.k * scale / softcap) (0: not capped) + rel[h, min(distance, last)] - slope[h] * distance;
    ``sink`` [H] adds exp(sink) to the denominator; with ``chunk`` position i only sees keys from i // chunk * chunk on, with
    ``window`` the keys i - window + 1 .. i.  ``wbias`` [H]: a key's weight is sigmoid(score + wbias) and nothing is normalised.
    ``turn``: cos and sin from :func:`head_store` (layout of halves) by which the heads' results are turned back; ``gate`` [T, H] (may
    be a column slice): results are multiplied by its sigmoid.  Returns [T, H * vdim]."""
    return _mixers(q).grouped_attention(q, keys, values, fb, kv_heads, scale, softcap, sink, rel, slope, chunk, window, wbias, turn,
                                        gate)


def conv_unit(p, taps, before, fb, heads: int, kv_heads: int, dim: int, vdim: int):
    """Short causal convolution per channel and silu over the q, k and v columns of p (each part starts at a multiple of
    eight columns), taps [n, channels], the inputs ahead of a portion from ``before`` [slots + 1, n - 1, channels]; then q and
    k as unit vectors, q times dim^-1/2.  Returns (q fp32 [T, kv_heads * dim], k, v [T, H * vdim]).  :func:`delta_rule` of the
    same layer must follow: it moves ``before`` on."""
    return _mixers(p).conv_unit(p, taps, before, fb, heads, kv_heads, dim, vdim)


def delta_rule(q, k, v, rate, dt_bias, a_log, p, at_b: int, gate, gain, eps: float, state, before, fb, heads: int,
               kv_heads: int):
    """Gated delta rule per head, S [dim, vdim] fp32 in ``state`` [slots + 1, H, dim, vdim]:

        S <- diag(g) S,  u = beta (v - S^T k),  S <- S + k u^T,  o = S^T q
        g = exp(-exp(a_log) softplus(rate + dt_bias)) per key channel,  beta = sigmoid(p[:, at_b + head])

    and y = o / rms(o) * gain * sigmoid(gate) per head -> [T, H * vdim].  Also keeps the last inputs of the convolutions
    (the q, k, v columns of p) in ``before``."""
    return _mixers(p).delta_rule(q, k, v, rate, dt_bias, a_log, p, at_b, gate, gain, eps, state, before, fb, heads, kv_heads)


# --------------------------------------------------------------------------- gated linear attention
def _gla(t):
    from . import cuda_gla, ref_gla

    return cuda_gla if t.is_cuda else ref_gla


def mlstm_gates(z, bias, cap: float, top, fb):
    """Exponential input gates with a running maximum: z fp32 [T, 2 H] (input gates, then forget gates), i = cap tanh((z + b) /
    cap), f = log sigmoid(cap tanh((z + b) / cap)), m = max(f + m, i) with m in ``top`` [slots + 1, H] (0 at the start of a
    sequence).  Returns (log of the decay f + m_before - m, factor of the keys e^(i - m), floor e^-m), each fp32 [T, H]."""
    return _gla(z).mlstm_gates(z, bias, cap, top, fb)


def causal_conv(p, taps, bias, before, fb):
    """silu of a short causal convolution per channel: p [T, C] (may be a column slice), taps [n, C] (the last row is the current
    token's), bias [C]; ``before`` [slots + 1, n - 1, C] holds the inputs ahead of a portion and is moved on.  Returns [T, C]."""
    return _gla(p).causal_conv(p, taps, bias, before, fb)


def gla(kind: str, q, k, v, gates, state, fb, heads: int, groups: int, q_mul: float = 1.0):
    """Gated linear attention per head, S <- diag(g) S + k v^T, o = S^T q, with S [d, columns] fp32 in ``state`` [slots + 1, H, d,
    columns]; v [T, H * e]; q, k [T, groups * d], shared by H / groups heads.  Gates by kind:

        "given"   (log g [T, H], factor of k [T, H]); the values have a column of ones at e
        "step"    (raw [T, H], bias [H], A_log [H]): dt = softplus(raw + bias), log g = -exp(A_log) dt, factor dt
        "forget"  (raw [T, H * d], bias [H * d], low [H * d]): g = low + (1 - low) sigmoid(raw + bias), k = 1 - g (k is None),
                  q goes through silu

    q is multiplied by ``q_mul``.  Returns o fp32 [T, H, columns]; columns from e on (e + 1 for "given") mean nothing."""
    return _gla(v).gla(kind, q, k, v, gates, state, fb, heads, groups, q_mul)


def norm_heads(o, e: int, gain, eps: float, dtype, gate=None, floor=None, mul: float = 1.0):
    """o [T, H, columns] -> o / rms(o) * gain * mul over the first e columns of every head (* sigmoid(gate)), as activations
    [T, H * e].  gain [e] or [H * e].  ``floor`` [T, H]: o is divided by max(|o[e]|, floor) + 1e-6 first."""
    return _gla(o).norm_heads(o, e, gain, eps, dtype, gate, floor, mul)


def norm_groups(o, skip, x, z, gain, groups: int, eps: float):
    """(o + skip x) silu(z) per head, then divided by the root mean square of each of ``groups`` equal parts, times gain.  o [T, H,
    columns] fp32, x and z [T, H * e] (may be column slices) -> [T, H * e]."""
    return _gla(o).norm_groups(o, skip, x, z, gain, groups, eps)


# --------------------------------------------------------------------------- sampling
def sample(logits, temperature, top_k, top_p, uniform, mask_ids=None):
    if logits.is_cuda:
        return _cu().sample(logits, temperature, top_k, top_p, uniform, mask_ids)
    return ref.sample(logits, temperature, top_k, top_p, uniform, mask_ids)


def argmax(logits):
    if logits.is_cuda:
        return _cu().argmax(logits)
    return logits.argmax(-1)
