"""Shared pieces of the tests of the layered designs: forwards over a shuffled page table, and traces through the engine."""
import torch

from minisgl.models.base import ForwardBatch


def make_fb(segs, device, ps=16, num_slots=6, max_len=2048, seed=0, prefill=True, pages=None):
    """segs: [(slot, first position, tokens)].  Every slot owns randomly placed pages; returns (fb, cache rows)."""
    g = torch.Generator().manual_seed(seed)
    per = -(-max_len // ps)
    pages = pages or per * (num_slots + 1)
    perm = torch.randperm(pages, generator=g)[: per * (num_slots + 1)].view(num_slots + 1, per)
    table = (perm[:, :, None] * ps + torch.arange(ps)).reshape(num_slots + 1, per * ps).to(torch.int32)
    pos = torch.cat([torch.arange(a, a + n) for _, a, n in segs]).to(torch.int32)
    slots = torch.cat([torch.full((n,), s) for s, _, n in segs]).to(torch.int32)
    lens = [n for _, _, n in segs]
    off = torch.tensor([0] + lens).cumsum(0).to(torch.int32)
    loc = table[slots.long(), pos.long()]
    to = lambda t: t.to(device)
    fb = ForwardBatch(to(torch.zeros_like(pos)), to(pos), to(slots), to(loc), None, to(table), prefill,
                      max(a + n for _, a, n in segs))
    if prefill:
        fb.seg_off, fb.seg_lens = to(off), lens
        fb.seg_ends, fb.seg_slots = [a + n for _, a, n in segs], [s for s, _, _ in segs]
    else:
        assert all(n == 1 for n in lens)
    return fb, pages * ps


def replay(engine_trace, requests, schedule):
    """requests: name -> token list; schedule: steps of [(name, tokens)].  Feeds them through a TraceReplay, asking for
    every logit; returns name -> [tokens, vocab].  A request ends when all its tokens have run."""
    at = {n: 0 for n in requests}
    out = {n: [] for n in requests}
    for step in schedule:
        entries = [{"id": n, "tokens": requests[n][at[n]:at[n] + k], "want": list(range(k))} for n, k in step]
        for n, k in step:
            at[n] += k
        got = engine_trace.step(entries, [n for n, _ in step if at[n] == len(requests[n])])
        lo = 0
        for n, k in step:
            out[n].append(got[lo:lo + k])
            lo += k
    return {n: torch.cat(v) for n, v in out.items() if v}


def mixed_schedule(requests, live, sizes, seed=0):
    """Random steps over the requests, at most ``live`` at a time, portions drawn from ``sizes``; some steps leave a live
    request out."""
    g = torch.Generator().manual_seed(seed)
    pick = lambda n: int(torch.randint(0, n, (1,), generator=g))
    left = {n: len(t) for n, t in requests.items()}
    waiting, active, steps = list(requests), [], []
    while waiting or active:
        while waiting and len(active) < live and (not active or pick(2)):
            active.append(waiting.pop(0))
        step = []
        for n in active:
            if len(active) > 1 and pick(5) == 0:
                continue
            step.append((n, min(sizes[pick(len(sizes))], left[n])))
        for n, k in step:
            left[n] -= k
        active = [n for n in active if left[n]]
        if step:
            steps.append(step)
    return steps
