"""The Sakevik design through the engine on CPU tensors, against the plain model: configuration and loader, cache and state across
portions, batches, page and slot reuse, generation, the trace runner."""
import copy
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import plain_sakevik as P
import sakevik_cases as K
from layered_util import replay
from minisgl.core import SamplingParams
from minisgl.kvcache import layered_pool
from minisgl.llm import LLM
from minisgl.models import sakevik_weight as W
from minisgl.models.layered_config import RotaryScaling, rotary_frequencies
from minisgl.models.registry import family_of, parse_config
from minisgl.models.sakevik_config import SakevikConfig

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(params=sorted(K.MODELS))
def case(request, tmp_path):
    return K.Case(request.param, tmp_path, "cpu", torch.float32)


@pytest.fixture
def mixed(tmp_path):
    return K.Case("mixed", tmp_path, "cpu", torch.float32)


# --------------------------------------------------------------------------- the plain model itself
def test_plain_model_steps_and_whole_agree():
    cfg = K.MODELS["mixed"]
    m = P.PlainSakevik(cfg, P.tensors(cfg))
    toks = K.tokens(cfg, 60, 1)
    want = m.step(toks)
    m.reset()
    assert K.rel_err(torch.cat([m.step(toks[:7]), *[m.step([t]) for t in toks[7:]]]), want) < 1e-10


def test_plain_rotation_depends_on_distance_only():
    g = torch.Generator().manual_seed(0)
    q, k = (torch.randn(1, 1, 12, generator=g, dtype=P.F) for _ in range(2))
    f = torch.tensor([0.9, 0.3, 0.01], dtype=P.F)
    for halves in (True, False):
        dot = lambda a, b: float((P.turn(q, torch.tensor([a]), f, 1.0, halves) * P.turn(k, torch.tensor([b]), f, 1.0, halves)).sum())
        assert abs(dot(7, 3) - dot(104, 100)) < 1e-9 and abs(dot(7, 3) - dot(7, 4)) > 1e-3
        back = P.turn(P.turn(q, torch.tensor([9]), f, 1.0, halves), torch.tensor([9]), f, 1.0, halves, back=True)
        assert K.rel_err(back[0], q[0]) < 1e-12


# --------------------------------------------------------------------------- configuration and weights
def test_configuration_round_trip():
    for raw in K.MODELS.values():
        cfg = parse_config(raw)
        assert isinstance(cfg, SakevikConfig) and family_of(cfg).name == "sakevik"
        assert parse_config(cfg.to_dict()) == cfg
        assert len(cfg.run_stores()) == len(raw["layers"]) == len(cfg.runs)
    cfg = parse_config({**K.MODELS["mixed"], "eos_token_id": 5, "max_position_embeddings": 99})
    assert cfg.max_position == 99 and cfg.eos_token_id == 5


def test_unknown_parts_are_refused():
    def changed(**change):
        raw = copy.deepcopy(K.MODELS["mixed"])
        for path, value in change.items():
            at = raw
            *way, last = [int(p) if p.isdigit() else p for p in path.split("__")]
            for p in way:
                at = at[p]
            at[last] = value
        return raw

    for change, text in (({"layers__0__type": "other"}, "unknown"), ({"layers__0__mlp__kind": "moe"}, "unknown"),
                         ({"layers__1__mixer__kv_heads": 4}, "evenly"), ({"layers__1__mixer__mask__size": 0}, "window"),
                         ({"layers__1__mixer__rot__dims": 34}, "rotary"), ({"layers__1__mixer__vdim": 7}, "pairs"),
                         ({"layers__2__mixer__rot__dims": 8}, "rotary"), ({"embedding__bigram__buckets": 0}, "bucket"),
                         ({"layers": []}, "layer")):
        with pytest.raises(ValueError, match=text):
            parse_config(changed(**change))


def test_loader_checks_names_and_shapes(tmp_path):
    raw = K.MODELS["mixed"]
    cfg, tens = parse_config(raw), P.tensors(raw)
    assert set(W.raw_shapes(cfg)) == set(tens)
    w = W.build_weights(cfg, tens.__getitem__, "cpu")
    # heads of 24 unrotated and 16 rotated rows are sorted, the latent's rows stand behind them
    q = tens["l2.mix.q"].view(4, 40, -1)
    assert torch.equal(w["l2.mix.qc"][24:48], q[1, :24]) and torch.equal(w["l2.mix.qc"][96 + 16:96 + 32], q[1, 24:])
    assert torch.equal(w["l2.mix.qc"][160:224], tens["l2.mix.dkv"])
    # an expanded key: the projected latent, then the turned part as it is cached
    c = torch.randn(3, 64, dtype=torch.float64)
    k = (c @ w["l2.mix.uk"].double().T).view(3, 4, 40)
    assert torch.equal(k[:, 2, 24:], c[:, 48:]) and torch.allclose(k[..., :24].reshape(3, -1), c[:, :48] @ tens["l2.mix.uk"].double().T)
    assert w["l1.mix.qkvg"].shape == (6 * 32 + 3 * 32 + 3 * 24 + 8, 96)       # the gates' six rows padded to eight
    bad = dict(tens, **{"l1.mix.o": tens["l1.mix.o"][:, :-1]})
    with pytest.raises(ValueError, match="l1.mix.o"):
        W.build_weights(cfg, bad.__getitem__, "cpu")
    del tens["final.norm"]
    with pytest.raises(KeyError, match="final.norm"):
        W.load_checkpoint(P.write_model(raw, tens, tmp_path), cfg, "cpu")


def test_random_weights_have_the_checkpoint_layout():
    for name in ("mixed", "ragged"):
        cfg = parse_config(K.MODELS[name])
        a, b = W.random_weights(cfg, "cpu", 3), W.build_weights(cfg, P.tensors(K.MODELS[name]).__getitem__, "cpu")
        assert {k: (v.shape, v.dtype) for k, v in a.items()} == {k: (v.shape, v.dtype) for k, v in b.items()}


@pytest.mark.parametrize("dims,base,scaling", [(64, 10000.0, None), (2, 7.0, None), (64, 150000.0, (4.0, 4096, 32.0, 1.0)),
                                               (16, 3000.0, (4.0, 64, 8.0, 1.0)), (24, 500.0, (1.5, 30, 1.0, 0.9)), (8, 9.0, (8.0, 10, 64.0, 32.0))])
def test_rotary_frequencies(dims, base, scaling):
    rot = {"base": base, "scaling": dict(zip(("factor", "original", "fast", "slow"), scaling)) if scaling else None}
    want, want_mul = P.frequencies(rot, dims)
    got, mul = rotary_frequencies(dims, base, RotaryScaling(*scaling) if scaling else None)
    assert torch.allclose(got.double(), want, rtol=1e-6, atol=0) and mul == pytest.approx(want_mul)
    if scaling:
        assert mul == pytest.approx(0.1 * math.log(scaling[0]) + 1.0)


def test_storage():
    cfg = parse_config(K.MODELS["mixed"])
    stores = cfg.run_stores()
    assert [k[0] for _, k in layered_pool.kinds(stores)] == ["tokens", "vector", "kv", "latent", "vector", "kv"]
    row = 3 * (32 + 24) + (48 + 16) + (16 + 64)
    assert layered_pool.bytes_per_page(stores, 16, torch.bfloat16) == 16 * (2 * row + 4)
    assert layered_pool.bytes_per_req_slot(stores, 96, torch.bfloat16) == 4 * (80 + 56)


# --------------------------------------------------------------------------- whole models
def test_layers_one_by_one(case):
    toks = K.tokens(case.cfg, 60, 5)
    t = case.trace(64)
    seen = []
    t.engine.model.on_run = lambda n, x: seen.append(x.clone())
    replay(t, {"a": toks}, [[("a", 60)]])
    case.want(toks)
    assert len(seen) == len(case.plain.residuals)
    for n, (got, want) in enumerate(zip(seen, case.plain.residuals)):
        assert K.rel_err(got, want) < 2e-5, n


def test_schedules(case):
    K.check_schedules(case)


def test_mixed_batches_reuse_pages_and_slots(case):
    K.check_mixed(case)


def test_batch_independence(mixed):
    K.check_batch_independence(mixed)


def test_generation(case):
    K.check_generation(case)


def test_bf16_activations(tmp_path):
    c = K.Case("mixed", tmp_path, "cpu", torch.bfloat16)
    c.run(K.portions([50, 3]), {"a": K.tokens(c.cfg, 90, 6)}, 128, "bf16")


def test_recurrent_layers_turn_prefix_reuse_off(mixed):
    llm, _, _ = K.check_generation(mixed)
    assert llm.cache.radix is None
    llm.engine.pool.assert_no_leak()


def test_prefixes_are_reused_without_recurrent_layers(tmp_path):
    """The pages of a prefix hold everything a later request needs, the token ahead of its first own one included."""
    llm, _ = K.shared_prefixes(K.Case("attention", tmp_path, "cpu", torch.float32))
    assert llm.cache.radix is not None and llm.engine.pool.prefix_reusable
    llm.shutdown()


def test_sampling_and_stop_token(mixed):
    kw = dict(device="cpu", page_size=16, max_running_req=2, num_page_override=16, context_length=128, disable_log_stats=True)
    llm = LLM(mixed.folder, mixed.dtype, **kw)
    prompt = K.tokens(mixed.cfg, 9, 8)
    greedy = llm.generate([prompt], SamplingParams(max_tokens=6))[0].token_ids
    assert llm.generate([prompt], SamplingParams(temperature=5.0, top_p=1e-6, max_tokens=6))[0].token_ids == greedy
    raw = {**mixed.cfg, "eos_token_id": greedy[2]}
    stop = LLM(P.write_model(raw, mixed.tensors, mixed.folder + "/stop"), mixed.dtype, **kw).generate([prompt], SamplingParams(max_tokens=6))[0]
    first = greedy.index(greedy[2])
    assert stop.token_ids == greedy[: first + 1] and stop.finish_reason == "stop"


# --------------------------------------------------------------------------- trace runner, command line
def test_trace_runner(mixed, tmp_path):
    out = tmp_path / "logits"
    out.mkdir()
    a, b = K.tokens(mixed.cfg, 12, 1), K.tokens(mixed.cfg, 5, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:8], "want": [7, 0]}, {"id": "b", "tokens": b[:2], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[2:], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[8:9], "want": [0]}], "end": []},
             {"step": 7, "entries": [{"id": "a", "tokens": a[9:], "want": [2]}], "end": ["a"]}]
    cmd = [sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", mixed.folder, "--dtype", "float32", "--out", str(out),
           "--max-tokens", "256", "--device", "cpu"]
    r = subprocess.run(cmd, input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 7"]
    want = mixed.want(a)
    for step, rows in ((0, [7, 0]), (2, [8]), (7, [11])):
        got = torch.frombuffer(bytearray((out / f"{step}.f32").read_bytes()), dtype=torch.float32).view(len(rows), -1)
        assert K.rel_err(got, want[rows]) < 1e-4


def test_command_line_serves_the_model(tmp_path):
    """``python -m minisgl``: the backend processes serve the design like any other model; the shell's answer is the plain
    model's greedy continuation."""
    from test_server_e2e_cpu import _write_tokenizer

    case = K.Case("single", tmp_path / "model", "cpu", torch.float32)
    _write_tokenizer(case.folder, case.cfg["vocab"])
    env = dict(os.environ, PYTHONPATH=ROOT + os.pathsep + os.environ.get("PYTHONPATH", ""), LOG_LEVEL="ERROR",
               MINISGL_SHELL_MAX_TOKENS="5", MINISGL_SHELL_TEMPERATURE="0.0")
    r = subprocess.run([sys.executable, "-m", "minisgl", "--model", case.folder, "--device", "cpu", "--dtype", "float32",
                        "--shell-mode", "--page-size", "16", "--num-pages", "16", "--context-length", "128"],
                       cwd=ROOT, env=env, input="w10 w11 w12\n/exit\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stdout[-1000:] + r.stderr[-2000:]
    ids = [10, 11, 12]
    for _ in range(5):
        case.plain.reset()
        ids.append(int(case.plain.step(ids)[-1].argmax()))
    names = {0: "<s>", 1: "</s>", 2: "<unk>", 3: "<think>", 4: "</think>"}
    assert " ".join(names.get(i, f"w{i}") for i in ids[3:]) in " ".join(r.stdout.split()), (ids, r.stdout)
