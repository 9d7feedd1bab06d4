"""Prefill and decode throughput of a layered design beside the closest other model at equal size: Bedalorn beside DeepSeek-V4,
Buvalix beside Bedalorn, Zazilix beside Bedalorn (whose experts are the like feed-forwards) and Buvalix (whose recurrence and
attention are the like mixers), Sakevik beside Buvalix (the like feed-forwards, attention and norms) and Bedalorn (the like latent
attention).

    python bench.py --design bedalorn|buvalix|zazilix|sakevik [--sizes small,large] [--profile]

Equal size: the same width, layer runs, attention heads, vocabulary and feed-forward weights (DeepSeek-V4: the same experts;
Buvalix's gated feed-forwards have three matrices, so the Bedalorn model beside it has dense ones half as wide again; Zazilix has
one expert less than the Bedalorn model with experts everywhere, and a shared one; Sakevik's windows of 1 024 and 2 048 positions
hold all of a short prompt), random weights, one GPU, through the offline API.  Per model and workload one JSON line: device time of the forwards (CUDA
events), tokens per second, and with ``--profile`` the per-launcher share of one eager forward of each phase.
Workloads: prefill forwards of 8 x 1 024 and 1 x 8 192 tokens; decode steps of 128 sequences at 1 024 tokens of context and
of 8 sequences at 8 192.
"""
from __future__ import annotations

import dataclasses
import json
import time

SIZES = {
    # width, attention heads, wkv heads, latent rank, dense ff, experts, top, expert ff, layers, loop passes, vocab
    "small": (2048, 16, 32, 512, 8192, 32, 4, 1024, 8, 1, 32768),
    "large": (4096, 32, 64, 512, 16384, 32, 4, 2048, 4, 2, 65536),
}
DENSE_SIZES = {
    # width, attention heads, key heads, delta heads, wkv heads, latent rank, gated ff, layers, loop passes, vocab
    "small": (2048, 16, 4, 16, 32, 512, 5632, 8, 1, 32768),
    "large": (4096, 32, 8, 32, 64, 512, 11264, 4, 2, 65536),
}
WORKLOADS = [("prefill", 8, 1024), ("prefill", 1, 8192), ("decode", 128, 1024), ("decode", 8, 8192)]


def _loop(n: int, passes: int):
    from minisgl.models.layered_config import LoopSpec

    return LoopSpec(0, n, passes) if passes > 1 else None


def bedalorn_config(size: str):
    from minisgl.models.bedalorn_config import BedalornConfig, DenseSpec, ExpertsSpec, LatentAttentionSpec, LayerSpec, WKVSpec

    d, h, hw, rank, ff, e, top, eff, n, passes, vocab = SIZES[size]
    attn = LatentAttentionSpec(h, 128, 128, rank, 128 ** -0.5)
    moe = ExpertsSpec(eff, e, top)
    layers = tuple(LayerSpec(WKVSpec(hw, 64), moe) if i % 4 == 2 else
                   LayerSpec(attn, DenseSpec(ff) if i % 4 == 0 else moe) for i in range(n))
    return BedalornConfig(layers, d, vocab, 1e-6, 1.0, _loop(n, passes), 1 << 17)


def bedalorn_dense_config(size: str):
    from minisgl.models.bedalorn_config import BedalornConfig, DenseSpec, LatentAttentionSpec, LayerSpec, WKVSpec

    d, h, _, _, hw, rank, ff, n, passes, vocab = DENSE_SIZES[size]
    attn = LatentAttentionSpec(h, 128, 128, rank, 128 ** -0.5)
    layers = tuple(LayerSpec(WKVSpec(hw, 64) if i % 4 == 2 else attn, DenseSpec(ff * 3 // 2)) for i in range(n))
    return BedalornConfig(layers, d, vocab, 1e-6, 1.0, _loop(n, passes), 1 << 17)


def buvalix_config(size: str):
    from minisgl.models.buvalix_config import (BuvalixConfig, ChannelDeltaSpec, DenseSpec, GroupedAttentionSpec, LayerSpec,
                                               QueryTemperature, RotarySpec)

    d, h, g, hd, _, _, ff, n, passes, vocab = DENSE_SIZES[size]
    rotary = GroupedAttentionSpec(h, g, 128, 128, 128 ** -0.5, 30.0, rot=RotarySpec(64, 1e5), bias=True, sink=True)
    bucket = GroupedAttentionSpec(h, g, 128, 128, 128 ** -0.5, 40.0, q_temp=QueryTemperature(0.1, 512), bias_max=2048)
    delta = ChannelDeltaSpec(hd, hd, 128, 128, 4)
    layers = tuple(LayerSpec((rotary, bucket, delta, rotary)[i % 4], DenseSpec(ff)) for i in range(n))
    return BuvalixConfig(layers, d, vocab, 1e-6, _loop(n, passes), 1 << 17)


def zazilix_config(size: str):
    from minisgl.models.layered_config import LayerSpec
    from minisgl.models.zazilix_config import (ChunkAttentionSpec, ForgetSpec, MambaSpec, MixtureSpec, MLSTMSpec, ParallelSpec,
                                               ZazilixConfig)

    d, h, _, _, _, e, top, eff, n, passes, vocab = SIZES[size]
    g, half = DENSE_SIZES[size][2], h // 2
    memory = MLSTMSpec(h, 128, 128, 15.0)
    both = ParallelSpec(ChunkAttentionSpec(h, g, 128, 128, 128 ** -0.5, 2048), ForgetSpec(half, 128, 128), 0.7, 0.7)
    mamba = MambaSpec(d // 32, 64, 8, 128, 4, 8)                      # twice the width inside
    ff = MixtureSpec(eff, e - 1, top - 1, 8, 1.0, eff)
    layers = tuple(LayerSpec((memory, both, mamba, both)[i % 4], ff) for i in range(n * passes))
    return ZazilixConfig(layers, d, vocab, 1e-6, 4, 1.0, 1 << 14, max_position=1 << 14)


def sakevik_config(size: str):
    from minisgl.models.layered_config import LayerSpec, RotaryScaling
    from minisgl.models.sakevik_config import (ClampedSpec, MinGRUSpec, PairEmbeddingSpec, RotarySpec, SakevikConfig,
                                               SigmoidAttentionSpec, WindowLatentSpec)

    d, h, g, _, _, rank, ff, n, passes, vocab = DENSE_SIZES[size]
    sigmoid = SigmoidAttentionSpec(h, g, 128, 128, 128 ** -0.5, 1024, RotarySpec(128, 1e5))
    latent = WindowLatentSpec(h, 96, 32, 128, rank, 128 ** -0.5, 2048, RotarySpec(32, 1e5, RotaryScaling(8.0, 4096, 32.0, 1.0)))
    layers = tuple(LayerSpec((sigmoid, latent, MinGRUSpec(d), sigmoid)[i % 4], ClampedSpec(ff, 7.0)) for i in range(n * passes))
    return SakevikConfig(layers, d, vocab, 1e-6, 1.0, PairEmbeddingSpec(4 * vocab, 31, 17), 1.0, max_position=1 << 17)


def bedalorn_experts_config(size: str):
    from minisgl.models.bedalorn_config import BedalornConfig, ExpertsSpec, LatentAttentionSpec, LayerSpec, WKVSpec

    d, h, hw, rank, _, e, top, eff, n, passes, vocab = SIZES[size]
    attn, moe = LatentAttentionSpec(h, 128, 128, rank, 128 ** -0.5), ExpertsSpec(eff, e, top)
    layers = tuple(LayerSpec(WKVSpec(hw, 64) if i % 4 in (0, 2) else attn, moe) for i in range(n * passes))
    return BedalornConfig(layers, d, vocab, 1e-6, 1.0, None, 1 << 17)


def dsv4_config(size: str):
    from minisgl.models.config import ModelConfig

    d, h, _, _, _, e, top, eff, n, passes, vocab = SIZES[size]
    return dataclasses.replace(ModelConfig.flash().with_layers(n * passes), hidden_size=d, num_heads=h, vocab_size=vocab,
                               n_routed_experts=e, num_experts_per_tok=top, moe_intermediate_size=eff, n_hash_layers=0,
                               o_groups=min(8, h // 4))


def _engine(cfg, batch: int, context: int, profile: bool):
    from minisgl.llm import LLM

    return LLM(model_config=cfg, use_dummy_weight=True, max_running_req=batch, context_length=context,
               cuda_graph_bs=[batch], cuda_graph_max_bs=0 if profile else batch, disable_log_stats=True,
               memory_ratio=0.8, cache_type="none")


def _decode_once(llm, batch: int, context: int) -> None:
    """One eager decode forward of ``batch`` sequences at ``context`` tokens (whatever the cache holds)."""
    import torch

    from minisgl.core import Batch, Req, SamplingParams

    reqs = []
    for i in range(batch):
        r = Req(torch.zeros(context, dtype=torch.int32), llm.table.allocate(), context - 1, 1, i, SamplingParams())
        for upto in range(256, context + 256, 256):    # window storage follows, as it does while a prompt is prefilled
            r.cached_len = min(upto, context) - 1
            llm.cache.allocate(r, min(upto, context))
            llm.cache.release_swa_behind(r)
        reqs.append(r)
    llm.engine.last_token.copy_(torch.randint(0, llm.engine.model_config.vocab_size, llm.engine.last_token.shape))
    b = Batch(reqs, "decode")
    llm._prepare_batch(b)
    llm.engine.forward_batch(b, llm.engine.sampler.prepare(b))
    torch.cuda.synchronize()


def _forward_ms(eng, phase: str, tokens: int):
    ms = sorted(t["events"][0].elapsed_time(t["events"][1]) for t in eng.timings
                if t["phase"] == phase and t["tokens"] == tokens)
    return (ms[len(ms) // 2], len(ms)) if ms else (None, 0)


def run(cfg, phase: str, batch: int, context: int, profile: bool, steps: int = 32) -> dict:
    import torch

    from minisgl.core import SamplingParams
    from minisgl.ops import native

    # decode: under mixed load four decode forwards run per 2 048-token prefill forward, so the first sequences are that
    # far into their output when the last prompt is done and the whole batch decodes together
    n_out = 1 if phase == "prefill" else 4 * -(-batch * context // 2048) + steps
    llm = _engine(cfg, batch, context + n_out + 64, profile)
    eng = llm.engine
    g = torch.Generator().manual_seed(7)

    def prompts():
        return [torch.randint(0, cfg.vocab_size, (context,), generator=g, dtype=torch.int32) for _ in range(batch)]

    llm.generate(prompts() if phase == "prefill" else [prompts()[0][:64]], SamplingParams(max_tokens=4, ignore_eos=True))
    eng.record_timings = True
    t0 = time.perf_counter()
    for _ in range(5 if phase == "prefill" else 1):
        llm.generate(prompts(), SamplingParams(max_tokens=n_out, ignore_eos=True))
    tokens = batch * context if phase == "prefill" else batch
    torch.cuda.synchronize()
    wall = time.perf_counter() - t0
    ms, n = _forward_ms(eng, phase, tokens)
    out = {"phase": phase, "sequences": batch, "context": context, "ms_per_forward": round(ms, 4), "forwards": n,
           "tok_s": round(tokens / ms * 1e3, 1), "wall_s": round(wall, 2), "weight_gib": round(eng.weight_bytes / 2**30, 2)}
    if profile:
        eng.record_timings = False
        native.enable_profile(True)
        if phase == "prefill":
            llm.generate(prompts(), SamplingParams(max_tokens=1, ignore_eos=True))
        else:
            _decode_once(llm, batch, context)
        rep = native.profile_report()
        native.enable_profile(False)
        out["share_ms"] = {k: [c, round(t, 3)] for k, (c, t) in list(rep.items())[:16]}
    native.assert_device_ok()
    llm.shutdown()
    return out


PAIRS = {
    "bedalorn": {"bedalorn": bedalorn_config, "dsv4": dsv4_config},
    "buvalix": {"buvalix": buvalix_config, "bedalorn": bedalorn_dense_config},
    "zazilix": {"zazilix": zazilix_config, "bedalorn": bedalorn_experts_config, "buvalix": buvalix_config},
    "sakevik": {"sakevik": sakevik_config, "buvalix": buvalix_config, "bedalorn": bedalorn_dense_config},
}


def main(design: str, sizes=("small", "large"), profile: bool = False, workloads=None) -> None:
    import gc

    import torch

    for size in sizes:
        for name, make in PAIRS[design].items():
            for phase, batch, context in workloads or WORKLOADS:
                r = run(make(size), phase, batch, context, profile)
                print(json.dumps({"design": name, "size": size, **r}), flush=True)
                gc.collect()
                torch.cuda.empty_cache()
