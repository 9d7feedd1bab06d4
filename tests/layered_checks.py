"""Checks of the engine against a plain model that hold for every layered design and run on any device: schedules of given
tokens, mixed batches over few pages and slots, generation, long decoding, far tokens."""
import torch

from layered_util import mixed_schedule, replay
from minisgl.core import SamplingParams
from minisgl.llm import LLM
from minisgl.trace import TraceReplay

F = torch.float64


def rel_err(got, want):
    """Root mean square difference over the root mean square of what is wanted, worst row."""
    got, want = got.to(F).cpu(), want.to(F)
    d = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt().clamp_min(1e-12)
    return float(d.max()) if d.numel() else 0.0


def tokens(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


class Case:
    """A small model in a folder, and its plain statement (``step(tokens)``, ``reset()``, ``residuals``).  limit: relative
    error a position may have; stray: share of the positions that may be further off (up to ``worst``)."""

    def __init__(self, cfg, tensors, plain, folder, device, dtype, limit, stray=0.0, worst=0.5):
        self.cfg, self.tensors, self.plain, self.folder = cfg, tensors, plain, folder
        self.device, self.dtype, self.limit, self._want = device, dtype, limit, {}
        self.stray, self.worst = stray, worst if stray else limit

    def trace(self, max_tokens, **kw):
        return TraceReplay(self.folder, self.dtype, max_tokens, device=self.device, **kw)

    def want(self, toks):
        key = tuple(toks)
        if key not in self._want:
            self.plain.reset()
            self._want[key] = self.plain.step(toks)
        return self._want[key]

    def check(self, got, toks, what=""):
        self.compare(got, self.want(toks)[: len(got)], what)

    def compare(self, got, want, what=""):
        e = torch.tensor([rel_err(g[None], w[None]) for g, w in zip(got, want)])
        stray = max(1, int(self.stray * len(e))) if self.stray else 0
        assert int((e >= self.limit).sum()) <= stray and float(e.max()) < self.worst, \
            (what, e.topk(min(8, len(e))))

    def run(self, schedule_of, requests, max_tokens, what):
        t = self.trace(max_tokens)
        out = replay(t, requests, schedule_of(requests))
        for n, toks in requests.items():
            self.check(out[n], toks, (what, n))
        t.engine.pool.assert_no_leak()
        assert t.table.available_size == t.engine.config.max_running_req and not t.live
        t.shutdown()
        return out


def whole(requests):
    return [[(n, len(t))] for n, t in requests.items()]


def token_by_token(prompt):
    def steps(requests):
        return [s for n, t in requests.items()
                for s in [[(n, min(prompt, len(t)))]] + [[(n, 1)]] * (len(t) - min(prompt, len(t)))]
    return steps


def portions(sizes):
    def steps(requests):
        out = []
        for n, t in requests.items():
            left, i = len(t), 0
            while left:
                k = min(sizes[i % len(sizes)], left)
                out.append([(n, k)])
                left, i = left - k, i + 1
        return out
    return steps


def check_schedules(case):
    """The same tokens whole, decoded one by one from the first and from a late position, and in portions whose edges fall
    on, before and behind page borders."""
    cfg = case.cfg
    reqs = {"a": tokens(cfg, 150, 1), "b": tokens(cfg, 1, 2), "c": tokens(cfg, 67, 3)}
    case.run(whole, reqs, 192, "whole")
    case.run(token_by_token(1), {"a": reqs["a"][:80], "b": reqs["b"]}, 128, "decode")
    case.run(token_by_token(100), {"a": reqs["a"]}, 192, "late decode")
    case.run(portions([2, 3, 61, 1, 64, 63]), reqs, 192, "portions")
    case.run(portions([2]), {"c": reqs["c"]}, 128, "pairs")


def check_mixed(case):
    """Unequal requests together, portions beside single tokens, requests that pause; the pool holds fewer pages and slots
    than all requests need, so both are used again."""
    cfg = case.cfg
    reqs = {f"r{i}": tokens(cfg, n, 10 + i) for i, n in enumerate((90, 3, 140, 40, 65, 1, 70, 130))}
    case.run(lambda r: mixed_schedule(r, 4, (1, 1, 1, 2, 5, 64, 33)), reqs, 11 * 64, "mixed")


def check_batch_independence(case):
    """Each request's logits do not depend on what else is in the batch."""
    cfg = case.cfg
    reqs = {"a": tokens(cfg, 70, 21), "b": tokens(cfg, 9, 22), "c": tokens(cfg, 64, 23)}
    t = case.trace(4 * 128)
    together = replay(t, reqs, [[("a", 70), ("b", 8), ("c", 63)], [("b", 1), ("c", 1)]])
    for n, toks in reqs.items():
        alone = replay(t, {n: toks}, [[(n, len(toks))]])[n]
        case.compare(together[n], alone.to(F), n)
        case.check(together[n], toks, n)
    t.shutdown()


def check_generation(case, **kw):
    """Greedy generation through the offline API and the scheduler: prompts prefilled in small portions beside decoding
    requests, more requests than slots.  Every generated token must be the plain model's choice, up to near ties."""
    llm = LLM(case.folder, case.dtype, device=case.device, page_size=16, max_running_req=3, num_page_override=40,
              max_extend_tokens=32, max_prefill_length=32, context_length=256, disable_log_stats=True, **kw)
    prompts = [tokens(case.cfg, n, 30 + n) for n in (45, 1, 17, 80, 33)]
    outs = llm.generate(prompts, SamplingParams(max_tokens=12, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert len(o.token_ids) == 12
        want = case.want(p + o.token_ids)
        for i, tok in enumerate(o.token_ids):
            row = want[len(p) - 1 + i]
            assert float(row.max() - row[tok]) <= 2 * case.limit * float(row.pow(2).mean().sqrt()), (len(p), i)
    assert llm.table.available_size == 3 and not llm.decode.running
    llm.shutdown()
    return llm, prompts, outs


def check_long_decode(case, n=600):
    """Hundreds of decoded tokens: positions far past the prompt, states carried through every step."""
    toks = tokens(case.cfg, n, 40)
    case.run(token_by_token(5), {"a": toks}, -(-n // 64) * 64, "long decode")


def check_far_key(case):
    """A token deep in the prompt decides a late logit: changing one far token changes the late logits as the plain model
    says, in a prompt and when the late tokens are decoded."""
    cfg = case.cfg
    base = tokens(cfg, 130, 50)
    for far in (0, 63, 64, 127):
        toks = list(base)
        toks[far] = (toks[far] + 1) % cfg["vocab"]
        for steps in (whole, token_by_token(129)):
            case.run(steps, {"a": toks}, 192, ("far", far))
