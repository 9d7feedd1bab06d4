"""The Zazilix design through the engine on CPU tensors, against the plain model: configuration and loader, cache and state across
portions, batches, page and slot reuse, generation, the trace runner."""
import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import plain_zazilix as P
import zazilix_cases as K
from layered_util import replay
from minisgl.core import SamplingParams
from minisgl.kvcache import layered_pool
from minisgl.llm import LLM
from minisgl.models import zazilix_weight as W
from minisgl.models.registry import family_of, parse_config
from minisgl.models.zazilix_config import ZazilixConfig

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
    m = P.PlainZazilix(cfg, P.tensors(cfg))
    toks = K.tokens(cfg, 60, 1)
    want = m.step(toks)
    m.reset()
    assert K.rel_err(torch.cat([m.step(toks[:7]), *[m.step([t]) for t in toks[7:]]]), want) < 1e-10


def test_plain_memory_does_not_depend_on_its_running_maximum():
    """The same recurrence without the maximum, on gates small enough for it."""
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(12, 2, n, generator=g, dtype=P.F) for n in (5, 5, 3))
    i, f = torch.randn(12, 2, generator=g, dtype=P.F), -torch.rand(12, 2, generator=g, dtype=P.F)
    zero = (torch.zeros(2, 5, 3, dtype=P.F), torch.zeros(2, 5, dtype=P.F), torch.zeros(2, dtype=P.F))
    got, (_, _, m) = P.mlstm_recurrence(q, k, v, i, f, zero)
    s, n = zero[0], zero[1]
    for t in range(12):
        keep, write = torch.exp(f[t]), torch.exp(i[t])
        s = keep[:, None, None] * s + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        top = (s * q[t][:, :, None]).sum(1)
        want = top / torch.maximum((n * q[t]).sum(-1).abs(), torch.ones(2, dtype=P.F))[:, None]
        assert K.rel_err(got[t], want) < 1e-4          # but for the 1e-6 in the denominator


# --------------------------------------------------------------------------- configuration and weights
def test_configuration_round_trip():
    for raw in K.MODELS.values():
        cfg = parse_config(raw)
        assert isinstance(cfg, ZazilixConfig) and family_of(cfg).name == "zazilix"
        assert parse_config(cfg.to_dict()) == cfg
        assert len(cfg.run_stores()) == len(raw["layers"]) == len(cfg.runs)
    cfg = parse_config(K.MODELS["mixed"])
    assert cfg.max_position == cfg.position_rows == 1024 and cfg.eos_token_id == -1
    assert parse_config({**K.MODELS["mixed"], "eos_token_id": 5, "max_position_embeddings": 99}).max_position == 99
    assert parse_config({**K.MODELS["mixed"], "max_position_embeddings": 9999}).max_position == 1024
    raw = copy.deepcopy(K.MODELS["mixed"])
    del raw["layers"][0]["mlp"]["router"]["identity"]
    assert parse_config(raw).layers[0].ff.identity == 0


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

    for change, text in (({"layers__0__type": "other"}, "unknown"), ({"layers__0__mlp__kind": "dense"}, "unknown"),
                         ({"layers__0__mixer__gate_cap": 0.0}, "gate_cap"), ({"layers__0__mlp__router__top": 99}, "chosen"),
                         ({"layers__1__mixer__left__kv_heads": 4}, "evenly"), ({"layers__1__mixer__left__mask__size": 0}, "chunk"),
                         ({"layers__2__mixer__groups": 3}, "evenly"), ({"layers__2__mixer__norm_groups": 7}, "parts"),
                         ({"layers__2__mixer__conv": 9}, "taps")):
        with pytest.raises(ValueError, match=text):
            parse_config(changed(**change))


def test_loader_checks_names_and_shapes(tmp_path):
    raw = K.MODELS["single"]
    cfg, tens = parse_config(raw), P.tensors(raw)
    assert set(W.raw_shapes(cfg)) == set(tens)
    w = W.build_weights(cfg, tens.__getitem__, "cpu")
    assert torch.equal(w["l0.hc1.pre"], torch.cat([tens["l0.hc1.in"], tens["l0.norm1"][None]]).float())
    assert w["l2.mix.in"].shape == (8 + 24, 48) and torch.equal(w["l2.mix.dt"], tens["l2.mix.in"][-1:])
    assert w["l0.mlp.shared.gu"].shape == (64, 48) and w["l0.mlp.shared.down"].shape == (48, 32)
    bad = dict(tens, **{"l0.mix.left.o": tens["l0.mix.left.o"][:, :-1]})
    with pytest.raises(ValueError, match="l0.mix.left.o"):
        W.build_weights(cfg, bad.__getitem__, "cpu")
    del tens["final.norm"]
    with pytest.raises(KeyError, match="final.norm"):
        W.load_checkpoint(P.write_model(raw, tens, tmp_path), cfg, "cpu")


def test_random_weights_have_the_checkpoint_layout():
    for name in ("mixed", "ragged"):
        cfg = parse_config(K.MODELS[name])
        a, b = W.random_weights(cfg, "cpu", 3), W.build_weights(cfg, P.tensors(K.MODELS[name]).__getitem__, "cpu")
        assert {k: (v.shape, v.dtype) for k, v in a.items()} == {k: (v.shape, v.dtype) for k, v in b.items()}


def test_slopes():
    for h in (1, 3, 8, 20):
        assert torch.allclose(W.slopes(h).to(P.F), torch.tensor(P.slopes(h), dtype=P.F), rtol=1e-7)


def test_storage_of_a_run_with_two_kinds():
    cfg = parse_config(K.MODELS["mixed"])
    stores = cfg.run_stores()
    assert [k[0] for _, k in layered_pool.kinds(stores)] == ["linear", "kv", "linear", "linear", "kv", "linear"]
    # keys and values of layers 1 and 3
    assert layered_pool.bytes_per_page(stores, 16, torch.bfloat16) == 16 * 2 * (3 * (16 + 24) + 1 * (24 + 16))
    slot = 3 * 24 * 20 + 3 + 2 * 24 * 32 + 4 * 16 * 24 + 3 * 16 * 8           # states and running maxima
    assert layered_pool.bytes_per_req_slot(stores, 96, torch.float32) == 4 * (slot + 2 * (4 * 24 + 2 * 2 * 16))


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


def test_sequences_end_with_the_learned_positions(tmp_path):
    """A longer context asked for on the command line does not reach past the table of position vectors."""
    cfg = {**K.MODELS["single"], "max_positions": 70}
    folder = P.write_model(cfg, P.tensors(cfg), tmp_path)
    llm = LLM(folder, torch.float32, device="cpu", page_size=16, max_running_req=2, num_page_override=40, context_length=512,
              disable_log_stats=True)
    assert llm.engine.max_seq_len == 70
    out = llm.generate([K.tokens(cfg, 60, 1)], SamplingParams(max_tokens=50, ignore_eos=True))[0]
    assert len(out.token_ids) == 10
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
