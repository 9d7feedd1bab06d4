"""Configuration of the Bedalorn design: a list of layers, each with its own mixer (latent attention or recurrent time
mixing) and feed-forward (dense, mixture of experts, or none), and an optional range of layers that runs several times
with the same weights."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .layered_config import DenseSpec, LayeredConfig, LayerSpec, LoopSpec, parse_loop, serving_limits

ARCHITECTURE = "Bedalorn"


@dataclass(frozen=True)
class LatentAttentionSpec:
    heads: int
    dim: int          # query / key dimensions per head
    vdim: int         # value dimensions per head
    kv_rank: int
    scale: float


@dataclass(frozen=True)
class WKVSpec:
    heads: int
    dim: int


@dataclass(frozen=True)
class ExpertsSpec:
    ff: int
    experts: int
    top: int


@dataclass(frozen=True)
class BedalornConfig(LayeredConfig):
    layers: Tuple[LayerSpec, ...]
    hidden_size: int
    vocab_size: int
    norm_eps: float
    logit_scale: float
    loop: Optional[LoopSpec] = None
    max_position: int = 1 << 20      # positions enter no computation: a limit of the page table, not of the design
    eos_token_id: int = -1           # none unless the configuration names one
    bos_token_id: int = -1
    architectures: tuple = (ARCHITECTURE,)
    model_type: str = "bedalorn"
    window_size: int = 0

    def mixer_store(self, mixer: Any) -> tuple:
        latent = isinstance(mixer, LatentAttentionSpec)
        return ("latent", mixer.kv_rank) if latent else ("state", mixer.heads, mixer.dim)

    # ------------------------------------------------------------------ config.json
    @staticmethod
    def from_dict(raw: Dict[str, Any]) -> "BedalornConfig":
        if raw.get("architecture") != ARCHITECTURE:
            raise ValueError(f"architecture {raw.get('architecture')!r} is not {ARCHITECTURE}")
        layers = tuple(_layer(i, e) for i, e in enumerate(raw["layers"]))
        return BedalornConfig(
            layers=layers, hidden_size=int(raw["width"]), vocab_size=int(raw["vocab"]),
            norm_eps=float(raw["norm"]["eps"]), logit_scale=float(raw["logit_scale"]),
            loop=parse_loop(raw, len(layers)), **serving_limits(raw, 1 << 20))

    def to_dict(self) -> Dict[str, Any]:
        """The inverse of from_dict."""
        def mlp(f):
            if f is None:
                return None
            if isinstance(f, DenseSpec):
                return {"kind": "dense", "ff": f.ff}
            return {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}}

        def layer(s):
            latent = isinstance(s.mixer, LatentAttentionSpec)
            return {"type": "latent_attention" if latent else "wkv", "mixer": dict(vars(s.mixer)), "mlp": mlp(s.ff)}

        return {"architecture": ARCHITECTURE, "layers": [layer(s) for s in self.layers], "width": self.hidden_size,
                "vocab": self.vocab_size, "norm": {"eps": self.norm_eps}, "logit_scale": self.logit_scale,
                "loop": dict(vars(self.loop)) if self.loop else None, "max_position_embeddings": self.max_position}


def _layer(i: int, e: Dict[str, Any]) -> LayerSpec:
    m, kind, f = e["mixer"], e["type"], e.get("mlp")
    if kind == "latent_attention":
        mixer = LatentAttentionSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), int(m["kv_rank"]), float(m["scale"]))
    elif kind == "wkv":
        mixer = WKVSpec(int(m["heads"]), int(m["dim"]))
    else:
        raise ValueError(f"layer {i}: unknown mixer {kind!r}")
    if f is None:
        return LayerSpec(mixer, None)
    if f["kind"] == "dense":
        return LayerSpec(mixer, DenseSpec(int(f["ff"])))
    if f["kind"] == "moe":
        r = f["router"]
        return LayerSpec(mixer, ExpertsSpec(int(f["expert"]["ff"]), int(r["experts"]), int(r["top"])))
    raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")
