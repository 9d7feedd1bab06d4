"""Replays a trace of given token ids through the engine, step by step, and returns logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N      (steps on standard input)

Nothing is sampled, everything else is the serving path: requests are admitted to table slots, their pages come from the
cache manager, every step is one prepared batch (portions of prompts beside single tokens; a step of single tokens only
is a decode batch and replays the captured graph), and a request that ends gives its pages and its slot back.

A step is one JSON object on a line:
    {"step": 4, "entries": [{"id": "x", "tokens": [11, 2], "want": [1]}, {"id": "y", "tokens": [40]}], "end": ["y"]}
``want``: places among the entry's tokens whose logits are written (in order) to OUT/<step>.f32 as little-endian fp32
[wanted, vocab].  After every step the line "done <step>" is printed.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List, Sequence

import torch

from .core import Batch, Req, SamplingParams
from .parallel.info import DistributedInfo
from .scheduler.config import SchedulerConfig
from .scheduler.scheduler import Scheduler
from .utils.misc import div_ceil

PAGE_SIZE = 64
MAX_REQUESTS = 4      # requests that may be live at the same time


class TraceReplay(Scheduler):
    def __init__(self, model_path: str = "", dtype: torch.dtype = torch.bfloat16, max_tokens: int = 4096,
                 max_requests: int = MAX_REQUESTS, **kwargs):
        pages = max(div_ceil(max_tokens, PAGE_SIZE), 1)
        kw = dict(page_size=PAGE_SIZE, num_page_override=pages, context_length=pages * PAGE_SIZE,
                  max_running_req=max_requests, cuda_graph_max_bs=max_requests,
                  max_prefill_length=min(8192, max(pages - 1, 1) * PAGE_SIZE), cache_type="none", offline_mode=True,
                  disable_log_stats=True)
        kw.update(kwargs)
        super().__init__(SchedulerConfig(model_path=model_path, tp_info=DistributedInfo(0, 1), dtype=dtype, **kw))
        self.live: Dict[str, Req] = {}
        self._admissions = 0

    # ------------------------------------------------------------------ requests
    def _take_tokens(self, rid: str, tokens: Sequence[int]) -> Req:
        ids = torch.tensor(list(tokens), dtype=torch.int32)
        if len(ids) == 0:
            raise ValueError(f"request {rid!r}: an entry needs at least one token")
        if int(ids.min()) < 0 or int(ids.max()) >= self.engine.model_config.vocab_size:
            raise ValueError(f"request {rid!r}: token id outside the vocabulary")
        req = self.live.get(rid)
        if req is not None:
            req.extend_host(ids)
            return req
        room = self.engine.max_seq_len - len(ids)
        if room < 0:
            raise ValueError(f"request {rid!r} is longer than the cache")
        self._admissions += 1
        req = Req(input_ids=ids, table_idx=self.table.allocate(), cached_len=0, output_len=room, uid=self._admissions,
                  sampling_params=SamplingParams(ignore_eos=True))
        req.lifecycle.admission = self._admissions
        self.live[rid] = req
        return req

    def _finish(self, rid: str) -> None:
        req = self.live.pop(rid)
        req.lifecycle.end("trace")
        self.pending_retire.append(req)
        self._retire_ready()

    # ------------------------------------------------------------------ steps
    def step(self, entries: List[dict], end: Sequence[str] = ()) -> torch.Tensor:
        """Runs all entries as one batch; fp32 logits [wanted, vocab] on the host, in the order of entries and want."""
        reqs = [self._take_tokens(e["id"], e["tokens"]) for e in entries]
        if len({id(r) for r in reqs}) != len(reqs):
            raise ValueError("a request may appear once in a step")
        out = torch.empty(0, self.engine.model_config.vocab_size)
        if reqs:
            for r in reqs:
                self.cache.allocate(r, r.device_len)
            lens = [len(e["tokens"]) for e in entries]
            rows, at = [], 0
            for e, n in zip(entries, lens):
                rows += [at + int(w) for w in e.get("want", [])]
                at += n
            if all(n == 1 and r.cached_len > 0 for r, n in zip(reqs, lens)):
                batch = Batch(reqs, "decode")
                self.engine.force_tokens(torch.tensor([r.table_idx for r in reqs]),
                                         torch.tensor([int(e["tokens"][0]) for e in entries]))
            else:
                batch = Batch(reqs, "prefill")
                batch.chunk_lens, batch.is_final = lens, [True] * len(reqs)
            self._prepare_batch(batch)
            tickets = [r.lifecycle.launch() for r in reqs]
            out = self.engine.forward_logits(batch, rows).float().cpu()
            if self.engine.is_cuda:
                from .ops import native

                native.assert_device_ok()
            for r, t in zip(reqs, tickets):
                r.lifecycle.land(r.lifecycle.admission, t)
                r.cached_len = r.device_len
        for rid in end:
            self._finish(rid)
        return out


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token ids and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors weights")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], required=True)
    ap.add_argument("--out", required=True, help="folder for the logits, one <step>.f32 per step")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens the cache pool holds")
    ap.add_argument("--device", choices=["cuda", "cpu"], default="cuda")
    a = ap.parse_args(argv)
    dtype = getattr(torch, a.dtype)
    from .models.registry import family_of, parse_config
    from .utils.hf import cached_load_hf_config

    cfg = parse_config(cached_load_hf_config(a.model))
    if dtype not in family_of(cfg).dtypes:
        print(f"{family_of(cfg).name} models are not served in {a.dtype}", file=sys.stderr)
        return 3
    with torch.no_grad():
        run = TraceReplay(a.model, dtype, a.max_tokens, model_config=cfg, device=a.device)
        for line in iter(sys.stdin.readline, ""):
            if not line.strip():
                continue
            s = json.loads(line)
            logits = run.step(s.get("entries", []), s.get("end", []))
            if len(logits):
                data = logits.contiguous().numpy().astype("<f4").tobytes()
                with open(os.path.join(a.out, f"{s['step']}.f32"), "wb") as f:
                    f.write(data)
            print(f"done {s['step']}", flush=True)
        run.shutdown()
    return 0


if __name__ == "__main__":
    sys.exit(main())
