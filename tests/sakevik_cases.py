"""Whole-model cases of the Sakevik design: small configurations, checked with ``layered_checks``."""
import torch

import layered_checks
import plain_sakevik as P
from layered_checks import *  # noqa: F401,F403

MODELS = {
    # every mixer; feed-forwards behind some of them; windows that end inside pages
    "mixed": P.config([P.mingru_layer(ff=P.dense()), P.attention_layer(ff=P.dense(56, 0.8)), P.latent_layer(ff=P.dense(40, 2.0)),
                       P.mingru_layer(56), P.attention_layer(4, 1, 16, 64, 33, 16, 5000.0, 0.4)]),
    # recurrences only: nothing but the tokens is paged
    "recurrent": P.config([P.mingru_layer(120, P.dense(24)), P.mingru_layer(36), P.mingru_layer(64)], width=64, vocab=80, buckets=7),
    # attention only: pages can be shared between requests; windows of whole pages, longer than most sequences, and of one position
    "attention": P.config([P.latent_layer(2, 32, 8, 16, 24, 64, ff=P.dense(32, 0.5)), P.attention_layer(20, 2, 16, 32, 64, 8),
                           P.attention_layer(3, 3, 24, 8, 1, 24), P.latent_layer(5, 8, 24, 24, 64, 700, scale=0.1, scaling=(2.0, 300, 4.0, 2.0)),
                           P.attention_layer(34, 1, 8, 16, 500, 4, 100.0, 0.5)], width=128, vocab=96),
    # sizes of one
    "single": P.config([P.attention_layer(1, 1, 2, 2, 2, 2), P.mingru_layer(1), P.latent_layer(1, 1, 2, 1, 1, 3)], width=48, vocab=64,
                       buckets=1, mul_prev=3, mul_cur=5),
    # rows that do not start on 16 bytes, nothing a multiple of eight; factors beyond 32 bits
    "ragged": P.config([P.latent_layer(3, 7, 6, 5, 11, 21, ff=P.dense(21, 1.1)), P.attention_layer(6, 2, 10, 14, 23, 6),
                        P.mingru_layer(19, P.dense(13)), P.attention_layer(2, 2, 7, 6, 40, 4)], width=50, vocab=77, buckets=1009,
                       mul_prev=2654435761, mul_cur=40503),
    # heads wider than the prompt kernel takes, latents wider than a 64-row tile
    "wide": P.config([P.attention_layer(2, 1, 160, 144, 90, 64, scale=0.1), P.latent_layer(2, 64, 64, 48, 512, 80, scale=0.04), P.mingru_layer(300),
                      P.latent_layer(2, 96, 48, 136, 200, 50, scale=0.04), P.attention_layer(2, 2, 96, 320, 30, 96, scale=0.1)], width=72, vocab=88),
}
LIMIT = {torch.float32: 1e-4, torch.bfloat16: 5e-2}
# The stream enters the sub-layers unnormed and a norm stands behind them: where an output is a small difference its rounding is
# amplified, with every backend at the same places.
STRAY, WORST = 0.02, 0.2


class Case(layered_checks.Case):
    def __init__(self, name, folder, device, dtype, **change):
        cfg = {**MODELS[name], **change}
        if dtype == torch.bfloat16:
            cfg = {**cfg, "norm": {"eps": 0.05}}      # small vectors stay small
        tensors = P.tensors(cfg, seed=len(name))
        super().__init__(cfg, tensors, P.PlainSakevik(cfg, tensors), P.write_model(cfg, tensors, folder), device, dtype, LIMIT[dtype],
                         STRAY if dtype == torch.bfloat16 else 0.0, WORST)


def shared_prefixes(case):
    """Requests with a common beginning through the scheduler: later ones resume behind pages that earlier ones left, and the first
    token after them still finds the one before it.  Returns (llm, outputs)."""
    from minisgl.core import SamplingParams
    from minisgl.llm import LLM

    llm = LLM(case.folder, case.dtype, device=case.device, page_size=16, max_running_req=2, num_page_override=60, context_length=256,
              disable_log_stats=True)
    common = layered_checks.tokens(case.cfg, 48, 70)
    prompts = [common + layered_checks.tokens(case.cfg, n, 71 + n) for n in (9, 1, 20)]
    outs = []
    for p in prompts:
        o = llm.generate([p], SamplingParams(max_tokens=8, ignore_eos=True))[0]
        want = case.want(p + o.token_ids)
        for i, tok in enumerate(o.token_ids):
            row = want[len(p) - 1 + i]
            assert float(row.max() - row[tok]) <= 2 * case.limit * float(row.pow(2).mean().sqrt()), (len(p), i)
        outs.append(o.token_ids)
    return llm, outs
