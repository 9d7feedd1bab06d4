"""The model families this engine serves.  A family knows how to read its configuration, load or draw its weights, size
and build its KV pool and build its model; the engine, the scheduler and the command line only see this interface."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Callable, Dict, List, Optional, Tuple

import torch

from ..kvcache.paged import PoolSizes
from ..utils.misc import div_ceil
from .bedalorn_config import ARCHITECTURE as BEDALORN
from .bedalorn_config import BedalornConfig
from .buvalix_config import ARCHITECTURE as BUVALIX
from .buvalix_config import BuvalixConfig
from .config import ModelConfig
from .sakevik_config import ARCHITECTURE as SAKEVIK
from .sakevik_config import SakevikConfig
from .zazilix_config import ARCHITECTURE as ZAZILIX
from .zazilix_config import ZazilixConfig


@dataclass(frozen=True)
class KVBudget:
    """What the KV plan needs to know before the pool exists."""

    bytes_per_page: int
    fixed_bytes: int       # independent of the number of pages
    window_slots: int      # sliding-window slots to reserve (0: the family has no windows)
    min_pages: int


@dataclass(frozen=True)
class ModelFamily:
    name: str
    config_type: type
    parse: Callable[[Any], Any]
    dtypes: Tuple[torch.dtype, ...]                 # activation types the model can be served in
    max_tp: int
    load: Callable[..., Dict[str, torch.Tensor]]    # (folder, cfg, device, rank, size, moe_mode)
    draw: Callable[..., Dict[str, torch.Tensor]]    # (cfg, device, rank, size, moe_mode, seed, on_host)
    budget: Callable[..., KVBudget]                 # (cfg, engine config, dtype)
    pool: Callable[..., Any]                        # (cfg, PoolSizes, device, dtype)
    build: Callable[..., Any]                       # (cfg, weights, pool, comm, moe_mode, dtype)
    context_classes: Callable[[Any, int], List[int]]   # graph context classes below the limit
    kernel_set: Optional[str] = None                # ops/build.py: what a checkout without a built library compiles


# --------------------------------------------------------------------------- DeepSeek-V4
def _dsv4_load(folder, cfg, device, rank, size, moe_mode):
    from .weight import load_checkpoint

    return load_checkpoint(folder, cfg, device, rank, size, moe_mode)


def _dsv4_draw(cfg, device, rank, size, moe_mode, seed, on_host):
    from . import synth

    cuda = torch.device(device).type == "cuda"
    return synth.random_weights(cfg, device, rank, size, moe_mode, seed, fast_experts=cuda,
                                draw_on_host=cuda and on_host)


def swa_slot_plan(max_running_req: int, prefill_budget: int, page_size: int, window: int) -> int:
    """Sliding-window slots to reserve: the pages of one full prefill forward, one spare, and per running request its
    hard share (:func:`minisgl.scheduler.cache.slots_per_request`: window pages, the page being written, the step
    overlap scheduling keeps in flight) plus ``ceil(window / ps)`` for the tail of the cached path it locks in the
    prefix tree.  Admission divides the pool by the hard share (``CacheManager.request_capacity``); the tree's part is
    an allowance that keeps prefix-hit resume points alive and is given up first under pressure.
    (The reference reserves at least 8 per request, python/minisgl/engine/engine.py:569-584.)"""
    from ..scheduler.cache import slots_per_request

    per_req = slots_per_request(window, page_size) + div_ceil(window, page_size)
    return div_ceil(prefill_budget, page_size) + 1 + max_running_req * per_req


def _dsv4_budget(cfg, c, dtype) -> KVBudget:
    from ..kvcache import pool as P

    ps = c.page_size
    slots = swa_slot_plan(c.max_running_req, c.max_prefill_length, ps, cfg.window_size)
    fixed = slots * P.bytes_per_swa_slot(cfg, ps) + (c.max_running_req + 1) * P.bytes_per_req_slot(cfg)
    return KVBudget(P.bytes_per_page(cfg, ps), fixed, slots, div_ceil(c.max_prefill_length, ps) + 1)


def _dsv4_pool(cfg, sizes: PoolSizes, device, dtype):
    from ..kvcache.pool import DSV4KVPool

    return DSV4KVPool(cfg, sizes, device)


def _dsv4_build(cfg, weights, pool, comm, moe_mode, dtype):
    from .deepseek_v4 import DSV4Model

    return DSV4Model(cfg, weights, pool, comm, moe_mode)


def _dsv4_classes(cfg, limit: int) -> List[int]:
    from ..dsv4_release import DSV4_RELEASE

    return [c for c in (4 * cfg.index_topk, DSV4_RELEASE.graph_short_context) if c < limit]


# --------------------------------------------------------------------------- layered designs
def _layered_budget(cfg, c, dtype) -> KVBudget:
    from ..kvcache import layered_pool as P

    stores = cfg.run_stores()
    # a model without attention layers still counts pages (they bound the sequence lengths)
    return KVBudget(max(P.bytes_per_page(stores, c.page_size, dtype), 1),
                    (c.max_running_req + 1) * P.bytes_per_req_slot(stores, cfg.hidden_size, dtype), 0, 1)


def _layered_pool(cfg, sizes: PoolSizes, device, dtype):
    from ..kvcache.layered_pool import LayeredPool

    return LayeredPool(cfg.run_stores(), cfg.hidden_size, sizes, device, dtype)


def _layered_classes(cfg, limit: int) -> List[int]:
    # a class fixes how many ways the keys of a small decode batch are split
    return [c for c in (2048, 32768) if c < limit]


def _bedalorn_load(folder, cfg, device, rank, size, moe_mode):
    from .bedalorn_weight import load_checkpoint

    return load_checkpoint(folder, cfg, device)


def _bedalorn_draw(cfg, device, rank, size, moe_mode, seed, on_host):
    from .bedalorn_weight import random_weights

    return random_weights(cfg, device, seed)


def _bedalorn_build(cfg, weights, pool, comm, moe_mode, dtype):
    from .bedalorn import BedalornModel

    return BedalornModel(cfg, weights, pool, comm, moe_mode, dtype)


def _buvalix_load(folder, cfg, device, rank, size, moe_mode):
    from .buvalix_weight import load_checkpoint

    return load_checkpoint(folder, cfg, device)


def _buvalix_draw(cfg, device, rank, size, moe_mode, seed, on_host):
    from .buvalix_weight import random_weights

    return random_weights(cfg, device, seed)


def _buvalix_build(cfg, weights, pool, comm, moe_mode, dtype):
    from .buvalix import BuvalixModel

    return BuvalixModel(cfg, weights, pool, comm, moe_mode, dtype)


def _zazilix_load(folder, cfg, device, rank, size, moe_mode):
    from .zazilix_weight import load_checkpoint

    return load_checkpoint(folder, cfg, device)


def _zazilix_draw(cfg, device, rank, size, moe_mode, seed, on_host):
    from .zazilix_weight import random_weights

    return random_weights(cfg, device, seed)


def _zazilix_build(cfg, weights, pool, comm, moe_mode, dtype):
    from .zazilix import ZazilixModel

    return ZazilixModel(cfg, weights, pool, comm, moe_mode, dtype)


def _sakevik_load(folder, cfg, device, rank, size, moe_mode):
    from .sakevik_weight import load_checkpoint

    return load_checkpoint(folder, cfg, device)


def _sakevik_draw(cfg, device, rank, size, moe_mode, seed, on_host):
    from .sakevik_weight import random_weights

    return random_weights(cfg, device, seed)


def _sakevik_build(cfg, weights, pool, comm, moe_mode, dtype):
    from .sakevik import SakevikModel

    return SakevikModel(cfg, weights, pool, comm, moe_mode, dtype)


FAMILIES = {
    "DeepseekV4ForCausalLM": ModelFamily("deepseek_v4", ModelConfig, ModelConfig.from_hf, (torch.bfloat16,), 64,
                                         _dsv4_load, _dsv4_draw, _dsv4_budget, _dsv4_pool, _dsv4_build, _dsv4_classes),
    BEDALORN: ModelFamily("bedalorn", BedalornConfig, BedalornConfig.from_dict, (torch.bfloat16, torch.float32), 1,
                          _bedalorn_load, _bedalorn_draw, _layered_budget, _layered_pool, _bedalorn_build,
                          _layered_classes, "layered"),
    BUVALIX: ModelFamily("buvalix", BuvalixConfig, BuvalixConfig.from_dict, (torch.bfloat16, torch.float32), 1,
                         _buvalix_load, _buvalix_draw, _layered_budget, _layered_pool, _buvalix_build,
                         _layered_classes, "grouped"),
    ZAZILIX: ModelFamily("zazilix", ZazilixConfig, ZazilixConfig.from_dict, (torch.bfloat16, torch.float32), 1,
                         _zazilix_load, _zazilix_draw, _layered_budget, _layered_pool, _zazilix_build,
                         _layered_classes, "streams"),
    SAKEVIK: ModelFamily("sakevik", SakevikConfig, SakevikConfig.from_dict, (torch.bfloat16, torch.float32), 1,
                         _sakevik_load, _sakevik_draw, _layered_budget, _layered_pool, _sakevik_build,
                         _layered_classes, "windows"),
}


def parse_config(raw: Any):
    """config.json (dict) or a PretrainedConfig -> the configuration of the family it names."""
    get = raw.get if isinstance(raw, dict) else lambda k, d=None: getattr(raw, k, d)
    name = get("architecture") or next(iter(get("architectures") or []), None)
    family = FAMILIES.get(name)
    # an unknown architecture gets the complaint of the oldest family
    return family.parse(raw) if family is not None else ModelConfig.from_hf(raw)


def family_of(cfg: Any) -> ModelFamily:
    for f in FAMILIES.values():
        if isinstance(cfg, f.config_type):
            return f
    raise TypeError(f"no model family for a configuration of type {type(cfg).__name__}")
