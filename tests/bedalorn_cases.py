"""Whole-model cases of the Bedalorn design: small configurations, checked with ``layered_checks``."""
import torch

import layered_checks
import plain_bedalorn as P
from layered_checks import *  # noqa: F401,F403

MODELS = {
    # every mechanism, a loop over the middle layers, a layer without feed-forward
    "mixed": P.config([P.attention_layer(mlp=P.dense()), P.wkv_layer(mlp=P.moe()),
                       P.attention_layer(heads=2, dim=32, vdim=24, kv_rank=56, scale=0.3), P.wkv_layer(3, 24, P.dense(40)),
                       P.attention_layer(5, 8, 16, 32, 0.4, P.moe(7, 3, 24))], loop={"start": 1, "stop": 4, "times": 3}),
    # the recurrence first and last, all layers looped; every expert is chosen, so that no close call of a router, carried on
    # by the state, blurs the comparison in bf16
    "state": P.config([P.wkv_layer(2, 16, P.moe(3, 3, 16)), P.attention_layer(mlp=None), P.wkv_layer(1, 32, P.dense(24))],
                      width=64, vocab=80, loop={"start": 0, "stop": 3, "times": 2}, logit_scale=0.7),
    # no loop; sizes of one
    "single": P.config([P.attention_layer(1, 16, 16, 16, 0.25, P.moe(1, 1, 8)), P.wkv_layer(1, 8, None)], width=48,
                       vocab=64, logit_scale=1.0),
    # attention only, one pass through the loop, more heads than the row tile of the decode kernel
    "latent": P.config([P.attention_layer(20, 16, 24, 72, 0.3, P.dense(56)), P.attention_layer(17, 8, 8, 40, 0.5, P.dense(32))],
                       width=128, vocab=96, loop={"start": 1, "stop": 2, "times": 1}, logit_scale=2.5),
    # rows that do not start on 16 bytes, nothing a multiple of eight
    "ragged": P.config([P.attention_layer(3, 10, 14, 22, 0.3, P.moe(3, 2, 15)), P.wkv_layer(3, 9, P.dense(21))], width=50,
                       vocab=77, loop={"start": 0, "stop": 1, "times": 2}),
}
LIMIT = {torch.float32: 1e-4, torch.bfloat16: 3e-2}
# In bf16 a router can decide a close call the other way: the one model with experts in a loop of several passes gets a wider
# limit, and a few positions may be further off.
WIDE = {"mixed": 3.0}
STRAY = 0.05


class Case(layered_checks.Case):
    def __init__(self, name, folder, device, dtype):
        cfg = MODELS[name]
        tensors, bf16 = P.tensors(cfg, seed=len(name)), dtype == torch.bfloat16
        super().__init__(cfg, tensors, P.PlainBedalorn(cfg, tensors), P.write_model(cfg, tensors, folder), device, dtype,
                         LIMIT[dtype] * (WIDE.get(name, 1.0) if bf16 else 1.0), STRAY if bf16 else 0.0)
