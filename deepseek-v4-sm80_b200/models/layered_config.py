"""What the layered designs share in their configurations: a list of layers, each with a mixer and a feed-forward, and an
optional range of layers that runs several times with the same weights."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional


@dataclass(frozen=True)
class DenseSpec:
    ff: int


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


def serving_limits(raw: Dict[str, Any], max_position: int) -> Dict[str, int]:
    """Keys that serving reads and the designs themselves do not name: no stop token unless one is given."""
    tok = lambda k: int(raw[k]) if raw.get(k) is not None else -1
    return {"max_position": int(raw.get("max_position_embeddings") or max_position), "eos_token_id": tok("eos_token_id"),
            "bos_token_id": tok("bos_token_id")}
