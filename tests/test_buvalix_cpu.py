"""The Buvalix design through the engine on CPU tensors, against the plain model: configuration and loader, cache and state
across portions, batches, page and slot reuse, generation, prefix reuse, the trace runner."""
import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import buvalix_cases as K
import plain_buvalix as P
from layered_util import replay
from minisgl.core import SamplingParams
from minisgl.llm import LLM
from minisgl.models import buvalix_weight as W
from minisgl.models.buvalix_config import BuvalixConfig
from minisgl.models.layered_config import LoopSpec
from minisgl.models.config import ModelConfig
from minisgl.models.registry import family_of, parse_config

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
    m = P.PlainBuvalix(cfg, P.tensors(cfg))
    toks = K.tokens(cfg, 20, 1)
    want = m.step(toks)
    m.reset()
    assert P.rel_err(torch.cat([m.step(toks[:7]), *[m.step([t]) for t in toks[7:]]]), want) < 1e-10


# --------------------------------------------------------------------------- configuration and weights
def test_configuration_round_trip_and_order_of_runs():
    cfg = parse_config(K.MODELS["mixed"])
    assert isinstance(cfg, BuvalixConfig) and family_of(cfg).name == "buvalix"
    assert parse_config(cfg.to_dict()) == cfg
    assert cfg.loop == LoopSpec(1, 4, 3)
    assert [r.layer for r in cfg.runs] == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4]
    assert [r.enters for r in cfg.runs] == [None, 0, None, None, 1, None, None, 2, None, None, None]
    assert len(cfg.run_stores()) == 11
    assert [r.layer for r in parse_config(K.MODELS["single"]).runs] == [0, 1]
    assert parse_config({**K.MODELS["single"], "eos_token_id": 5}).eos_token_id == 5


def test_unknown_parts_are_refused():
    for change in ({"type": "other"}, {"mlp": {"kind": "other"}}):
        raw = copy.deepcopy(K.MODELS["single"])
        raw["layers"][0].update(change)
        with pytest.raises(ValueError, match="unknown"):
            parse_config(raw)
    with pytest.raises(ValueError, match="loop"):
        parse_config({**K.MODELS["single"], "loop": {"start": 0, "stop": 9, "times": 1}})
    with pytest.raises(ValueError):
        parse_config({"architecture": "Unheard"})
    assert isinstance(parse_config(ModelConfig.tiny().to_hf_dict()), ModelConfig)


def test_loader_checks_names_and_shapes(tmp_path):
    raw = K.MODELS["single"]
    cfg, tens = parse_config(raw), P.tensors(raw)
    assert set(W.raw_shapes(cfg)) == set(tens)
    w = W.build_weights(cfg, tens.__getitem__, "cpu")
    assert torch.equal(w["l0.norm1.b"], tens["l0.norm1.b"].float())
    gu = w["l0.mlp.gu"]          # blocks of 16 gate rows, 16 up rows; the feed-forward size padded to 32
    assert gu.shape == (64, 48) and torch.equal(gu[:16], tens["l0.mlp.gate"][:16]) and torch.equal(gu[16:32], tens["l0.mlp.up"][:16])
    assert torch.equal(gu[32:40], tens["l0.mlp.gate"][16:]) and float(gu[40:48].abs().max()) == 0
    bad = dict(tens, **{"l0.mix.o": tens["l0.mix.o"][:, :-1]})
    with pytest.raises(ValueError, match="l0.mix.o"):
        W.build_weights(cfg, bad.__getitem__, "cpu")
    del tens["final.norm"]
    with pytest.raises(KeyError, match="final.norm"):
        W.load_checkpoint(P.write_model(raw, tens, tmp_path), cfg, "cpu")


def test_random_weights_have_the_checkpoint_layout():
    cfg = parse_config(K.MODELS["delta"])
    raw = P.tensors(K.MODELS["delta"], rank=12, buckets=22)
    raw.update({k: v[:12] if k.endswith("g1") else v[:, :12] for k, v in raw.items() if k.endswith(("mix.g1", "mix.g2"))})
    a, b = W.random_weights(cfg, "cpu", 3, rank=12, buckets=20), W.build_weights(cfg, raw.__getitem__, "cpu")
    assert {k: (v.shape, v.dtype) for k, v in a.items()} == {k: (v.shape, v.dtype) for k, v in b.items()}


def test_engine_refuses_what_the_family_cannot_do(tmp_path):
    with pytest.raises(ValueError, match="served in"):
        LLM(model_config=ModelConfig.tiny(), dtype=torch.float32, device="cpu", use_dummy_weight=True)
    from minisgl.parallel.info import DistributedInfo

    with pytest.raises(ValueError, match="at most 1 GPU"):
        LLM(model_config=parse_config(K.MODELS["single"]), tp_info=DistributedInfo(0, 2), device="cpu", use_dummy_weight=True)


# --------------------------------------------------------------------------- whole models
def test_layers_one_by_one(case):
    toks = K.tokens(case.cfg, 40, 5)
    t = case.trace(64)
    seen = []
    t.engine.model.on_run = lambda n, x: seen.append(x.clone())
    replay(t, {"a": toks}, [[("a", 40)]])
    case.want(toks)
    assert len(seen) == len(case.plain.residuals)
    for n, (got, want) in enumerate(zip(seen, case.plain.residuals)):
        assert P.rel_err(got, want) < 2e-5, n


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


def test_prefix_reuse_without_recurrent_layers(tmp_path):
    case = K.Case("attention", tmp_path, "cpu", torch.float32)
    llm = LLM(case.folder, case.dtype, device="cpu", page_size=16, max_running_req=2, num_page_override=32,
              context_length=256, disable_log_stats=True)
    shared = K.tokens(case.cfg, 60, 7)
    sp = SamplingParams(max_tokens=5, ignore_eos=True)
    for tail in ([1, 2], [3]):
        o = llm.generate([shared + tail], sp)[0]
        want = case.want(shared + tail + o.token_ids)
        assert o.token_ids == [int(want[len(shared + tail) - 1 + i].argmax()) for i in range(5)]
    assert llm.cache.radix.metrics["hit_tokens"] == 48       # 60 shared tokens: three whole pages


def test_bucket_table_spread_over_distances():
    for rows, limit in ((20, 100), (32, 128), (8, 5000), (12, 7), (2, 3)):
        table = torch.randn(rows, 3)
        got = W.spread_buckets(table, limit)
        for n in (*range(300), limit - 1, limit, limit + 1, 10 * limit):
            assert torch.equal(got[:, min(n, got.shape[1] - 1)], table[P.distance_bucket(n, rows, limit)]), (rows, limit, n)


def test_recurrent_layers_turn_prefix_reuse_off(mixed):
    llm, _, _ = K.check_generation(mixed)
    assert llm.cache.radix is None
    llm.engine.pool.assert_no_leak()


def test_sampling_and_stop_token(mixed):
    kw = dict(device="cpu", page_size=16, max_running_req=2, num_page_override=16, context_length=128, disable_log_stats=True)
    llm = LLM(mixed.folder, mixed.dtype, **kw)
    prompt = K.tokens(mixed.cfg, 9, 8)
    greedy = llm.generate([prompt], SamplingParams(max_tokens=6))[0].token_ids
    nucleus = llm.generate([prompt], SamplingParams(temperature=5.0, top_p=1e-6, max_tokens=6))[0].token_ids
    assert nucleus == greedy
    hot = llm.generate([prompt] * 2, SamplingParams(temperature=50.0, max_tokens=6))
    assert len({tuple(o.token_ids) for o in hot}) == 2
    raw = {**mixed.cfg, "eos_token_id": greedy[2]}
    stop = LLM(P.write_model(raw, mixed.tensors, mixed.folder + "/stop"), mixed.dtype, **kw).generate([prompt], SamplingParams(max_tokens=6))[0]
    first = greedy.index(greedy[2])
    assert stop.token_ids == greedy[: first + 1] and stop.finish_reason == "stop"


# --------------------------------------------------------------------------- trace runner
def run_cli(folder, out, steps, dtype="float32", max_tokens=256):
    cmd = [sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out),
           "--max-tokens", str(max_tokens), "--device", "cpu"]
    return subprocess.run(cmd, input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)


def test_trace_runner(mixed, tmp_path):
    out = tmp_path / "logits"
    out.mkdir()
    a, b = K.tokens(mixed.cfg, 12, 1), K.tokens(mixed.cfg, 5, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:8], "want": [7, 0]}, {"id": "b", "tokens": b[:2], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[2:], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[8:9], "want": [0]}], "end": []},
             {"step": 7, "entries": [{"id": "a", "tokens": a[9:], "want": [2]}], "end": ["a"]}]
    r = run_cli(mixed.folder, out, steps)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 7"]
    assert sorted(os.listdir(out)) == ["0.f32", "2.f32", "7.f32"]
    want = mixed.want(a)
    for step, rows in ((0, [7, 0]), (2, [8]), (7, [11])):
        got = torch.frombuffer(bytearray((out / f"{step}.f32").read_bytes()), dtype=torch.float32).view(len(rows), -1)
        assert P.rel_err(got, want[rows]) < 1e-4


def test_trace_runner_refuses_a_type_the_model_has_not(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(ModelConfig.tiny().to_hf_dict()))
    assert run_cli(str(tmp_path), tmp_path, []).returncode == 3


def test_trace_rejects_bad_steps(mixed):
    t = mixed.trace(64)
    for entry in ({"id": "a", "tokens": []}, {"id": "a", "tokens": [mixed.cfg["vocab"]]}, {"id": "a", "tokens": [0] * 65}):
        with pytest.raises(ValueError):
            t.step([entry])


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
