"""Configuration of the Sakevik design: a list of layers whose mixer is an element-wise gated recurrence ("mingru"), attention in a
window whose weights are sigmoids, with values that turn with their positions ("attention"), or latent attention in a window
("latent_attention"); feed-forwards whose gate and up halves are clamped; norms on the sub-layers' outputs only; an embedding of
token pairs beside the tokens' own."""
from __future__ import annotations

from dataclasses import asdict, dataclass
from typing import Any, Dict, Optional, Tuple

from .layered_config import LayeredConfig, LayerSpec, LoopSpec, RotaryScaling, parse_scaling, serving_limits

ARCHITECTURE = "Sakevik"


@dataclass(frozen=True)
class MinGRUSpec:
    width: int


@dataclass(frozen=True)
class RotarySpec:
    dims: int                              # leading dimensions of a head that turn
    base: float
    scaling: Optional[RotaryScaling] = None


@dataclass(frozen=True)
class SigmoidAttentionSpec:
    heads: int
    kv_heads: int
    dim: int                               # query / key dimensions per head
    vdim: int                              # value dimensions per head
    scale: float
    window: int                            # positions seen, the query's own included
    rot: RotarySpec


@dataclass(frozen=True)
class WindowLatentSpec:
    heads: int
    dim: int                               # unrotated query / key dimensions per head
    rot_dim: int                           # rotated ones, shared by all key heads
    vdim: int
    kv_rank: int
    scale: float
    window: int
    rot: RotarySpec


@dataclass(frozen=True)
class ClampedSpec:
    ff: int
    limit: float


@dataclass(frozen=True)
class PairEmbeddingSpec:
    """Row (token before * mul_prev + token * mul_cur) mod buckets of a table; its last row begins a sequence."""

    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class SakevikConfig(LayeredConfig):
    layers: Tuple[LayerSpec, ...]
    hidden_size: int
    vocab_size: int
    norm_eps: float
    embedding_scale: float
    pairs: PairEmbeddingSpec
    logit_scale: float
    loop: Optional[LoopSpec] = None
    max_position: int = 1 << 20
    eos_token_id: int = -1           # none unless the configuration names one
    bos_token_id: int = -1
    architectures: tuple = (ARCHITECTURE,)
    model_type: str = "sakevik"
    window_size: int = 0

    def mixer_store(self, mixer: Any) -> tuple:
        if isinstance(mixer, MinGRUSpec):
            return ("vector", mixer.width)
        if isinstance(mixer, SigmoidAttentionSpec):
            return ("kv", mixer.kv_heads * mixer.dim, mixer.kv_heads * mixer.vdim)
        return ("latent", mixer.kv_rank + mixer.rot_dim)

    def run_stores(self) -> list:
        """The first run also keeps the tokens, for the embedding of pairs ahead of it."""
        first, *rest = super().run_stores()
        return [(("tokens",), first), *rest]

    # ------------------------------------------------------------------ config.json
    @staticmethod
    def from_dict(raw: Dict[str, Any]) -> "SakevikConfig":
        if raw.get("architecture") != ARCHITECTURE:
            raise ValueError(f"architecture {raw.get('architecture')!r} is not {ARCHITECTURE}")
        emb = raw["embedding"]
        pairs = PairEmbeddingSpec(**{n: int(emb["bigram"][n]) for n in ("buckets", "mul_prev", "mul_cur")})
        if pairs.buckets < 1:
            raise ValueError("embedding.bigram: at least one bucket")
        if not raw["layers"]:
            raise ValueError("a model has at least one layer")
        return SakevikConfig(
            layers=tuple(_layer(i, e) for i, e in enumerate(raw["layers"])), hidden_size=int(raw["width"]),
            vocab_size=int(raw["vocab"]), norm_eps=float(raw["norm"]["eps"]), embedding_scale=float(emb["scale"]), pairs=pairs,
            logit_scale=float(raw["logit_scale"]), **serving_limits(raw, 1 << 20))

    def to_dict(self) -> Dict[str, Any]:
        """The inverse of from_dict."""
        def layer(s):
            m, f = s.mixer, s.ff
            mixer = asdict(m)
            if isinstance(m, MinGRUSpec):
                kind = "mingru"
            else:
                kind = "attention" if isinstance(m, SigmoidAttentionSpec) else "latent_attention"
                mixer["mask"] = {"size": mixer.pop("window")}
                if m.rot.scaling is None:
                    mixer["rot"].pop("scaling")
            return {"type": kind, "mixer": mixer, "mlp": None if f is None else {"kind": "dense", "ff": f.ff, "limit": f.limit}}

        return {"architecture": ARCHITECTURE, "layers": [layer(s) for s in self.layers], "width": self.hidden_size,
                "vocab": self.vocab_size, "norm": {"eps": self.norm_eps}, "logit_scale": self.logit_scale,
                "embedding": {"scale": self.embedding_scale, "bigram": asdict(self.pairs)},
                "max_position_embeddings": self.max_position}


def _layer(i: int, e: Dict[str, Any]) -> LayerSpec:
    m, kind, f = e["mixer"], e["type"], e.get("mlp")
    if kind == "mingru":
        mixer = MinGRUSpec(int(m["width"]))
    elif kind in ("attention", "latent_attention"):
        rot = RotarySpec(int(m["rot"]["dims"]), float(m["rot"]["base"]), parse_scaling(m["rot"].get("scaling")))
        rest = dict(scale=float(m["scale"]), window=int(m["mask"]["size"]), rot=rot)
        if rest["window"] < 1:
            raise ValueError(f"layer {i}: a window has at least one position")
        ints = lambda *names: {n: int(m[n]) for n in names}
        if kind == "attention":
            mixer = SigmoidAttentionSpec(**ints("heads", "kv_heads", "dim", "vdim"), **rest)
            if mixer.heads % mixer.kv_heads:
                raise ValueError(f"layer {i}: {mixer.heads} heads do not share {mixer.kv_heads} key heads evenly")
            if rot.dims % 2 or rot.dims > mixer.dim:
                raise ValueError(f"layer {i}: {rot.dims} rotary dimensions do not fit heads of {mixer.dim}")
            if mixer.vdim % 2:
                raise ValueError(f"layer {i}: values of {mixer.vdim} dimensions do not turn in pairs")
        else:
            mixer = WindowLatentSpec(**ints("heads", "dim", "rot_dim", "vdim", "kv_rank"), **rest)
            if rot.dims != mixer.rot_dim or rot.dims % 2 or rot.dims < 2:
                raise ValueError(f"layer {i}: {rot.dims} rotary dimensions are not the {mixer.rot_dim} of the rotated part")
    else:
        raise ValueError(f"layer {i}: unknown mixer {kind!r}")
    if f is None:
        return LayerSpec(mixer, None)
    if f["kind"] != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")
    return LayerSpec(mixer, ClampedSpec(int(f["ff"]), float(f["limit"])))
