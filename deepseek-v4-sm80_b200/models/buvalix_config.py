"""Configuration of the Buvalix design: a list of layers whose mixer is causal attention with rotary positions and a sink
("attention"), causal attention with a query temperature and a learned distance bias ("attention_2"), or a gated delta rule
with one decay per key channel ("channel_delta"); gated feed-forwards; layer norms before and after every sub-layer; and an
optional range of layers that runs several times with the same weights."""
from __future__ import annotations

from dataclasses import asdict, dataclass
from typing import Any, Dict, Optional, Tuple

from .layered_config import DenseSpec, LayeredConfig, LayerSpec, LoopSpec, parse_loop, serving_limits

ARCHITECTURE = "Buvalix"


@dataclass(frozen=True)
class RotarySpec:
    dims: int         # leading dimensions of a head that turn, in neighbouring pairs
    base: float


@dataclass(frozen=True)
class QueryTemperature:
    coef: float
    every: int        # positions per step of the temperature


@dataclass(frozen=True)
class GroupedAttentionSpec:
    heads: int
    kv_heads: int
    dim: int                                   # query / key dimensions per head
    vdim: int                                  # value dimensions per head
    scale: float
    softcap: float                             # scores become softcap * tanh(score / softcap)
    rot: Optional[RotarySpec] = None
    q_temp: Optional[QueryTemperature] = None
    bias: bool = False                         # q, k and v have biases
    sink: bool = False                         # a learned logit per head in the denominator
    bias_max: int = 0                          # > 0: learned bias by distance, the last bucket begins before this


@dataclass(frozen=True)
class ChannelDeltaSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int                                  # taps of the short convolutions


@dataclass(frozen=True)
class BuvalixConfig(LayeredConfig):
    layers: Tuple[LayerSpec, ...]
    hidden_size: int
    vocab_size: int
    norm_eps: float
    loop: Optional[LoopSpec] = None
    max_position: int = 1 << 20
    eos_token_id: int = -1           # none unless the configuration names one
    bos_token_id: int = -1
    architectures: tuple = (ARCHITECTURE,)
    model_type: str = "buvalix"
    window_size: int = 0

    def mixer_store(self, mixer: Any) -> tuple:
        if isinstance(mixer, GroupedAttentionSpec):
            return ("kv", mixer.kv_heads * mixer.dim, mixer.kv_heads * mixer.vdim)
        channels = 2 * mixer.kv_heads * mixer.dim + mixer.heads * mixer.vdim
        return ("delta", mixer.heads, mixer.dim, mixer.vdim, channels, mixer.conv)

    # ------------------------------------------------------------------ config.json
    @staticmethod
    def from_dict(raw: Dict[str, Any]) -> "BuvalixConfig":
        if raw.get("architecture") != ARCHITECTURE:
            raise ValueError(f"architecture {raw.get('architecture')!r} is not {ARCHITECTURE}")
        layers = tuple(_layer(i, e) for i, e in enumerate(raw["layers"]))
        return BuvalixConfig(
            layers=layers, hidden_size=int(raw["width"]), vocab_size=int(raw["vocab"]),
            norm_eps=float(raw["norm"]["eps"]), loop=parse_loop(raw, len(layers)), **serving_limits(raw, 1 << 20))

    def to_dict(self) -> Dict[str, Any]:
        """The inverse of from_dict."""
        def layer(s):
            m = s.mixer
            if isinstance(m, ChannelDeltaSpec):
                kind, mixer = "channel_delta", asdict(m)
            else:
                kind = "attention_2" if m.bias_max else "attention"
                keep = ("heads", "kv_heads", "dim", "vdim", "scale", "softcap") \
                    + (("bias_max", "q_temp") if m.bias_max else ("rot",))
                mixer = {k: v for k, v in asdict(m).items() if k in keep}
            return {"type": kind, "mixer": mixer, "mlp": None if s.ff is None else {"kind": "dense", "ff": s.ff.ff}}

        return {"architecture": ARCHITECTURE, "layers": [layer(s) for s in self.layers], "width": self.hidden_size,
                "vocab": self.vocab_size, "norm": {"eps": self.norm_eps},
                "loop": asdict(self.loop) if self.loop else None, "max_position_embeddings": self.max_position}


def _layer(i: int, e: Dict[str, Any]) -> LayerSpec:
    m, kind, f = e["mixer"], e["type"], e.get("mlp")
    sizes = {k: int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim")}
    if sizes["heads"] % sizes["kv_heads"]:
        raise ValueError(f"layer {i}: {sizes['heads']} heads do not share {sizes['kv_heads']} key heads evenly")
    if kind == "attention":
        rot = RotarySpec(int(m["rot"]["dims"]), float(m["rot"]["base"]))
        if rot.dims % 2 or rot.dims > sizes["dim"]:
            raise ValueError(f"layer {i}: {rot.dims} rotary dimensions do not fit heads of {sizes['dim']}")
        mixer = GroupedAttentionSpec(**sizes, scale=float(m["scale"]), softcap=float(m["softcap"]), rot=rot, bias=True,
                                     sink=True)
    elif kind == "attention_2":
        t = m["q_temp"]
        if t["every"] != int(t["every"]) or t["every"] < 1 or m["bias_max"] < 1:
            raise ValueError(f"layer {i}: q_temp.every and bias_max are positive counts of positions")
        mixer = GroupedAttentionSpec(**sizes, scale=float(m["scale"]), softcap=float(m["softcap"]),
                                     q_temp=QueryTemperature(float(t["coef"]), int(t["every"])), bias_max=int(m["bias_max"]))
    elif kind == "channel_delta":
        mixer = ChannelDeltaSpec(**sizes, conv=int(m["conv"]))
    else:
        raise ValueError(f"layer {i}: unknown mixer {kind!r}")
    if f is None:
        return LayerSpec(mixer, None)
    if f["kind"] != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")
    return LayerSpec(mixer, DenseSpec(int(f["ff"])))
