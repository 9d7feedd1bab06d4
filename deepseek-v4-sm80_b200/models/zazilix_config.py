"""Configuration of the Zazilix design: a list of layers whose mixer is a matrix memory with exponential gates ("mlstm"), chunked
attention beside a gated recurrence ("parallel"), or a state-space recurrence ("mamba2"); feed-forwards that mix experts, inputs
passed on and a shared expert; several residual streams with constant mixing weights; learned position vectors."""
from __future__ import annotations

from dataclasses import asdict, dataclass
from typing import Any, Dict, Optional, Tuple

from .layered_config import LayeredConfig, LayerSpec, LoopSpec, serving_limits

ARCHITECTURE = "Zazilix"
MAX_TAPS = 8          # of the short convolutions


@dataclass(frozen=True)
class MLSTMSpec:
    heads: int
    dim: int
    vdim: int
    gate_cap: float                # gate logits become cap * tanh(logit / cap)


@dataclass(frozen=True)
class ChunkAttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int                     # positions of a chunk: keys of earlier chunks are not seen


@dataclass(frozen=True)
class ForgetSpec:
    heads: int
    dim: int
    vdim: int


@dataclass(frozen=True)
class ParallelSpec:
    left: ChunkAttentionSpec
    right: ForgetSpec
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class MambaSpec:
    heads: int
    vdim: int
    groups: int                    # of heads that share B and C
    state: int
    conv: int                      # taps of the short convolution
    norm_groups: int               # equal parts the output is normed in


@dataclass(frozen=True)
class MixtureSpec:
    ff: int
    experts: int
    top: int
    identity: int                  # further router outputs that stand for the input itself
    scale: float
    shared: int                    # size of the expert that every token uses


@dataclass(frozen=True)
class ZazilixConfig(LayeredConfig):
    layers: Tuple[LayerSpec, ...]
    hidden_size: int
    vocab_size: int
    norm_eps: float
    streams: int
    embedding_scale: float
    position_rows: int               # learned position vectors
    loop: Optional[LoopSpec] = None
    max_position: int = 0            # longest sequence (at most position_rows)
    eos_token_id: int = -1           # none unless the configuration names one
    bos_token_id: int = -1
    architectures: tuple = (ARCHITECTURE,)
    model_type: str = "zazilix"
    window_size: int = 0

    def mixer_store(self, mixer: Any) -> tuple:
        up4 = lambda n: -(-n // 4) * 4
        if isinstance(mixer, MLSTMSpec):
            return ("linear", mixer.heads, mixer.dim, up4(mixer.vdim + 1), mixer.heads, 0, 1)
        if isinstance(mixer, ParallelSpec):
            l, r = mixer.left, mixer.right
            return (("kv", l.kv_heads * l.dim, l.kv_heads * l.vdim), ("linear", r.heads, r.dim, up4(r.vdim), 0, 0, 1))
        channels = mixer.heads * mixer.vdim + 2 * mixer.groups * mixer.state
        return ("linear", mixer.heads, mixer.state, up4(mixer.vdim), 0, channels, mixer.conv)

    # ------------------------------------------------------------------ config.json
    @staticmethod
    def from_dict(raw: Dict[str, Any]) -> "ZazilixConfig":
        if raw.get("architecture") != ARCHITECTURE:
            raise ValueError(f"architecture {raw.get('architecture')!r} is not {ARCHITECTURE}")
        rows = int(raw["max_positions"])
        limits = serving_limits(raw, rows)
        limits["max_position"] = min(limits["max_position"], rows)
        return ZazilixConfig(
            layers=tuple(_layer(i, e) for i, e in enumerate(raw["layers"])), hidden_size=int(raw["width"]),
            vocab_size=int(raw["vocab"]), norm_eps=float(raw["norm"]["eps"]), streams=int(raw["streams"]),
            embedding_scale=float(raw["embedding"]["scale"]), position_rows=rows, **limits)

    def to_dict(self) -> Dict[str, Any]:
        """The inverse of from_dict."""
        def mlp(f):
            if f is None:
                return None
            return {"kind": "moe", "expert": {"ff": f.ff}, "shared": {"ff": f.shared},
                    "router": {"experts": f.experts, "top": f.top, "identity": f.identity, "scale": f.scale}}

        def layer(s):
            m = s.mixer
            if isinstance(m, ParallelSpec):
                left = asdict(m.left)
                left["mask"] = {"size": left.pop("chunk")}
                mixer = {"left": left, "right": asdict(m.right), "left_scale": m.left_scale, "right_scale": m.right_scale}
                return {"type": "parallel", "mixer": mixer, "mlp": mlp(s.ff)}
            return {"type": "mlstm" if isinstance(m, MLSTMSpec) else "mamba2", "mixer": asdict(m), "mlp": mlp(s.ff)}

        return {"architecture": ARCHITECTURE, "layers": [layer(s) for s in self.layers], "width": self.hidden_size,
                "vocab": self.vocab_size, "norm": {"eps": self.norm_eps}, "streams": self.streams,
                "embedding": {"scale": self.embedding_scale}, "max_positions": self.position_rows,
                "max_position_embeddings": self.max_position}


def _ints(raw: Dict[str, Any], *names: str) -> Dict[str, int]:
    return {n: int(raw[n]) for n in names}


def _layer(i: int, e: Dict[str, Any]) -> LayerSpec:
    m, kind, f = e["mixer"], e["type"], e.get("mlp")
    if kind == "mlstm":
        mixer = MLSTMSpec(**_ints(m, "heads", "dim", "vdim"), gate_cap=float(m["gate_cap"]))
        if mixer.gate_cap <= 0:
            raise ValueError(f"layer {i}: gate_cap is positive")
    elif kind == "parallel":
        l, r = m["left"], m["right"]
        left = ChunkAttentionSpec(**_ints(l, "heads", "kv_heads", "dim", "vdim"), scale=float(l["scale"]),
                                  chunk=int(l["mask"]["size"]))
        if left.heads % left.kv_heads:
            raise ValueError(f"layer {i}: {left.heads} heads do not share {left.kv_heads} key heads evenly")
        if left.chunk < 1:
            raise ValueError(f"layer {i}: a chunk has at least one position")
        mixer = ParallelSpec(left, ForgetSpec(**_ints(r, "heads", "dim", "vdim")), float(m["left_scale"]),
                             float(m["right_scale"]))
    elif kind == "mamba2":
        mixer = MambaSpec(**_ints(m, "heads", "vdim", "groups", "state", "conv", "norm_groups"))
        if mixer.heads % mixer.groups:
            raise ValueError(f"layer {i}: {mixer.heads} heads do not share {mixer.groups} groups evenly")
        if mixer.heads * mixer.vdim % mixer.norm_groups:
            raise ValueError(f"layer {i}: {mixer.heads * mixer.vdim} values do not fall into {mixer.norm_groups} equal parts")
        if not 1 <= mixer.conv <= MAX_TAPS:
            raise ValueError(f"layer {i}: convolutions have 1 to {MAX_TAPS} taps")
    else:
        raise ValueError(f"layer {i}: unknown mixer {kind!r}")
    if f is None:
        return LayerSpec(mixer, None)
    if f["kind"] != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")
    r = f["router"]
    ff = MixtureSpec(int(f["expert"]["ff"]), int(r["experts"]), int(r["top"]), int(r.get("identity") or 0), float(r["scale"]),
                     int(f["shared"]["ff"]))
    if not 1 <= ff.top <= ff.experts + ff.identity:
        raise ValueError(f"layer {i}: {ff.top} of {ff.experts + ff.identity} router outputs cannot be chosen")
    return LayerSpec(mixer, ff)
