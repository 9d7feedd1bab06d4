"""What the layered designs share in their configurations: a list of layers, each with a mixer and a feed-forward, and an
optional range of layers that runs several times with the same weights."""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

import torch


@dataclass(frozen=True)
class DenseSpec:
    ff: int


@dataclass(frozen=True)
class RotaryScaling:
    """YaRN: slow pairs (fewer than ``slow`` turns over ``original`` positions) turn ``factor`` times slower, fast ones as they are."""

    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class LayerSpec:
    mixer: Any
    ff: Any           # a feed-forward specification or None


@dataclass(frozen=True)
class LoopSpec:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class LayerRun:
    """One pass of one layer.  ``enters``: the number of the loop pass that begins right before it, or None."""

    layer: int
    enters: Optional[int] = None


class LayeredConfig:
    """Base of the configurations; subclasses are dataclasses with ``layers`` and ``loop``."""

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def runs(self) -> List[LayerRun]:
        """The layer runs of one forward, in order."""
        n, lp = len(self.layers), self.loop
        if lp is None:
            return [LayerRun(i) for i in range(n)]
        out = [LayerRun(i) for i in range(lp.start)]
        for t in range(lp.times):
            out += [LayerRun(i, t if i == lp.start else None) for i in range(lp.start, lp.stop)]
        return out + [LayerRun(i) for i in range(lp.stop, n)]

    def mixer_store(self, mixer: Any) -> tuple:
        raise NotImplementedError

    def run_stores(self) -> list:
        """What every run keeps between forwards (kvcache/layered_pool.py)."""
        return [self.mixer_store(self.layers[r.layer].mixer) for r in self.runs]


def parse_loop(raw: Dict[str, Any], n_layers: int) -> Optional[LoopSpec]:
    loop = raw.get("loop")
    if not loop:
        return None
    loop = LoopSpec(int(loop["start"]), int(loop["stop"]), int(loop["times"]))
    if not (0 <= loop.start < loop.stop <= n_layers and loop.times >= 1):
        raise ValueError(f"loop {loop} does not fit {n_layers} layers")
    return loop


def parse_scaling(raw: Optional[Dict[str, Any]]) -> Optional[RotaryScaling]:
    return RotaryScaling(**{n: float(raw[n]) for n in ("factor", "original", "fast", "slow")}) if raw else None


def rotary_frequencies(dims: int, base: float, scaling: Optional[RotaryScaling] = None) -> Tuple[torch.Tensor, float]:
    """(angle per position of each of the dims / 2 pairs, fp32; factor of cos and sin)."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = base ** (-2.0 * i / max(dims, 1))
    if scaling is None:
        return f.float(), 1.0
    s = scaling
    # the pair that makes so many turns over the original positions
    pair = lambda turns: dims * math.log(s.original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(pair(s.fast)), 0), min(math.ceil(pair(s.slow)), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return (f / s.factor * ramp + f * (1.0 - ramp)).float(), 0.1 * math.log(s.factor) + 1.0


def serving_limits(raw: Dict[str, Any], max_position: int) -> Dict[str, int]:
    """Keys that serving reads and the designs themselves do not name: no stop token unless one is given."""
    tok = lambda k: int(raw[k]) if raw.get(k) is not None else -1
    return {"max_position": int(raw.get("max_position_embeddings") or max_position), "eos_token_id": tok("eos_token_id"),
            "bos_token_id": tok("bos_token_id")}
