"""The Sakevik design through the engine on the GPU, in both serving types, against the plain model."""
import dataclasses

import pytest
import torch

import sakevik_cases as K
from layered_util import replay
from minisgl.core import SamplingParams
from minisgl.llm import LLM
from minisgl.ops import cuda_layers as CL
from minisgl.ops import cuda_mixers as C

pytestmark = pytest.mark.gpu
TYPES = {"bf16": torch.bfloat16, "fp32": torch.float32}


@pytest.fixture(params=[f"{m}-{t}" for m in sorted(K.MODELS) for t in TYPES])
def case(request, tmp_path):
    name, t = request.param.split("-")
    return K.Case(name, tmp_path, "cuda", TYPES[t])


@pytest.fixture(params=sorted(TYPES))
def mixed(request, tmp_path):
    return K.Case("mixed", tmp_path, "cuda", TYPES[request.param])


def test_layers_one_by_one(case):
    toks = K.tokens(case.cfg, 130, 5)
    t = case.trace(192)
    seen = []
    t.engine.model.on_run = lambda n, x: seen.append(x.clone())
    replay(t, {"a": toks}, [[("a", 130)]])
    case.want(toks)
    assert len(seen) == len(case.plain.residuals)
    for n, (got, want) in enumerate(zip(seen, case.plain.residuals)):
        case.compare(got, want, n)
        if case.dtype == torch.float32:
            d = (got.cpu().to(K.F) - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()
            assert float(d.median()) < 1e-5, (n, float(d.median()))


def test_schedules(case):
    K.check_schedules(case)


def test_mixed_batches_reuse_pages_and_slots(case):
    K.check_mixed(case)


def test_batch_independence(mixed):
    K.check_batch_independence(mixed)


def test_generation(case):
    K.check_generation(case)


@pytest.mark.parametrize("model", ["recurrent", "attention", "mixed"])
@pytest.mark.parametrize("dtype", sorted(TYPES))
def test_far_tokens(model, dtype, tmp_path):
    K.check_far_key(K.Case(model, tmp_path, "cuda", TYPES[dtype]))


@pytest.mark.parametrize("model", ["recurrent", "mixed"])
@pytest.mark.parametrize("dtype", sorted(TYPES))
def test_long_decode(model, dtype, tmp_path):
    K.check_long_decode(K.Case(model, tmp_path, "cuda", TYPES[dtype]))


@pytest.mark.parametrize("form", ["flash", "rows"])
def test_both_kernels_of_prefill_attention(form, tmp_path, monkeypatch):
    monkeypatch.setattr(C, "GROUPED_PREFILL", form)
    monkeypatch.setattr(CL, "LATENT_PREFILL", "expanded" if form == "flash" else "absorbed")
    case = K.Case("attention", tmp_path, "cuda", torch.bfloat16)
    K.check_schedules(case)
    K.check_mixed(case)


@pytest.mark.parametrize("dtype", sorted(TYPES))
def test_prefixes_are_reused_without_recurrent_layers(dtype, tmp_path):
    llm, _ = K.shared_prefixes(K.Case("attention", tmp_path, "cuda", TYPES[dtype]))
    assert llm.cache.radix is not None
    llm.shutdown()


def test_graph_replay_gives_the_eager_tokens(tmp_path):
    case = K.Case("mixed", tmp_path, "cuda", torch.bfloat16)
    _, _, a = K.check_generation(case)
    _, _, b = K.check_generation(case, cuda_graph_max_bs=0)
    assert [o.token_ids for o in a] == [o.token_ids for o in b]


@pytest.mark.parametrize("model", ["recurrent", "mixed"])
def test_poisoned_storage_changes_nothing(model, tmp_path):
    """Whatever pages and slots held before, a new request starts clean."""
    case = K.Case(model, tmp_path, "cuda", torch.bfloat16)
    reqs = {"a": K.tokens(case.cfg, 90, 3), "b": K.tokens(case.cfg, 1, 4)}

    def run(poison):
        t = case.trace(192)
        if poison:
            for x in t.engine.pool.storage():
                x.fill_(float("nan") if x.is_floating_point() else 17)
        out = replay(t, reqs, [[("a", 70), ("b", 1)], [("a", 3)], [("a", 1)]] + [[("a", 1)]] * 16)
        t.shutdown()
        return out

    a, b = run(False), run(True)
    assert all(torch.equal(a[n], b[n]) for n in reqs)


def test_model_of_serving_size_decodes_and_prefills():
    """Sizes of a real model's layers: wide rows, 128-dimensional heads, every kernel's full tiles."""
    from minisgl.benchmark.designs import sakevik_config

    full = sakevik_config("small")
    cfg = dataclasses.replace(full, layers=full.layers[:4], vocab_size=512)
    llm = LLM(model_config=cfg, use_dummy_weight=True, max_running_req=4, num_page_override=64, context_length=4096,
              disable_log_stats=True)
    g = torch.Generator().manual_seed(1)
    prompts = [torch.randint(0, 512, (n,), generator=g).tolist() for n in (700, 33, 1500)]
    sp = SamplingParams(max_tokens=6, ignore_eos=True)
    a = [o.token_ids for o in llm.generate(prompts, sp)]
    assert a == [o.token_ids for o in llm.generate(prompts, sp)] and all(len(t) == 6 for t in a)
    llm.shutdown()
