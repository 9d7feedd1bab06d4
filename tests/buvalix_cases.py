"""Whole-model cases of the Buvalix design: small configurations, checked with ``layered_checks``."""
import torch

import layered_checks
import plain_buvalix as P
from layered_checks import *  # noqa: F401,F403

MODELS = {
    # every mechanism, a loop over the middle layers, a layer without feed-forward
    "mixed": P.config([P.rotary_layer(), P.delta_layer(), P.bucket_layer(), P.delta_layer(6, 2, 20, 12, 4, 48),
                       P.rotary_layer(3, 1, 32, 16, 32, 900.0, 0.2, 30.0, None)], loop={"start": 1, "stop": 4, "times": 3}),
    # the recurrence first and last, all layers looped
    "delta": P.config([P.delta_layer(2, 2, 32, 16, 4, 40), P.bucket_layer(ff=None), P.delta_layer(3, 1, 16, 64, 2)],
                      width=64, vocab=80, loop={"start": 0, "stop": 3, "times": 2}),
    # no loop; sizes of one, a convolution of one tap
    "single": P.config([P.rotary_layer(1, 1, 16, 16, 2, 100.0, 0.3, 5.0, 24), P.delta_layer(1, 1, 8, 8, 1)], width=48, vocab=64),
    # attention only, one pass through the loop, more query heads to a key head than the decode kernel's smallest row tile
    "attention": P.config([P.rotary_layer(20, 1, 16, 24, 8, 1e4, 0.3, 8.0, 56), P.bucket_layer(34, 2, 8, 8, 130, 0.2, 16, 0.5, 4.0, 32),
                           P.bucket_layer(4, 4, 48, 40, 40, 0.5, 1, 0.2, 50.0, 64)], width=128, vocab=96,
                          loop={"start": 1, "stop": 2, "times": 1}),
    # rows that do not start on 16 bytes, nothing a multiple of eight
    "ragged": P.config([P.rotary_layer(3, 1, 10, 14, 6, 50.0, 0.3, 11.0, 21), P.delta_layer(3, 3, 9, 7, 3, 15),
                        P.bucket_layer(2, 2, 7, 9, 33, 0.3, 10, 0.4, 6.0, None)], width=50, vocab=77,
                       loop={"start": 0, "stop": 1, "times": 2}),
    # heads wider than the prompt kernel and the chunked recurrence take
    "wide": P.config([P.rotary_layer(2, 1, 160, 144, 64, 1e4, 0.1, 15.0, 40), P.delta_layer(2, 1, 136, 152, 4)], width=72, vocab=88),
}
LIMIT = {torch.float32: 1e-4, torch.bfloat16: 5e-2}
# Unit vectors and head norms of small vectors amplify rounding: in bf16 a few positions are further off, with every backend
# at the same places.
STRAY, WORST = 0.045, 0.16


class Case(layered_checks.Case):
    def __init__(self, name, folder, device, dtype):
        cfg = MODELS[name]
        tensors = P.tensors(cfg, seed=len(name))
        super().__init__(cfg, tensors, P.PlainBuvalix(cfg, tensors), P.write_model(cfg, tensors, folder), device, dtype,
                         LIMIT[dtype], STRAY if dtype == torch.bfloat16 else 0.0, WORST)
