"""Model families: which configuration class, weights, caches and decoder serve an architecture.

`config.json` names its architecture ("architecture", or the first entry of "architectures"); without one it is read as the
DeepSeek-V4 layout this engine started with.  A configuration object names its family (`cfg.family`), and everything the
engine, the server and the checkpoint reader build for a model goes through that family's entry here.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Any, Callable, Dict, Mapping, Optional, Tuple

import torch

from ..config import (ConfigError, EngineConfig, domilix_config_from_json, fanulix_config_from_json, fogizen_config_from_json,
                      model_config_from_hf, timalorn_config_from_json)


@dataclass(frozen=True)
class ModelFamily:
    name: str
    weight_shapes: Callable[[Any], Dict[str, Tuple[Tuple[int, ...], str]]]
    build_weights: Callable[..., Any]          # (cfg, source, device, tp_rank, tp_size, layer_range) -> weights
    make_cache: Callable[..., Any]             # (engine cfg, device, context, comm, tp_rank, pipe) -> cache manager
    make_model: Callable[..., Any]             # (engine cfg, weights, cache, comm, tp_rank) -> Decoder
    prefix_cache: bool                         # prefixes can be kept and adopted
    # cfg -> (name, .cu files) of the library that holds just the kernels its steps need; None: the whole library
    native_sources: Optional[Callable[[Any], Tuple[str, Tuple[str, ...]]]] = None


# ---- DeepSeek-V4-style -----------------------------------------------------------------------
def _dsv4_shapes(cfg):
    from .weights import weight_shapes
    return weight_shapes(cfg)


def _dsv4_weights(cfg, src, device, tp_rank=0, tp_size=1, layer_range=None):
    from .dsv4 import build_model_weights
    return build_model_weights(cfg, src, device, tp_rank, tp_size,
                               head_fp8=cfg.dense_dtype == "fp8" and torch.device(device).type == "cuda", layer_range=layer_range)


def _dsv4_cache(cfg: EngineConfig, device, ctx: int, comm, tp_rank: int, pipe):
    from ..runtime.kv import KVManager, memory_pool_tokens, size_pools
    sc = cfg.sched
    # decode context parallel: the ranks of the tensor-parallel group each store 1/dcp of the ratio-4 caches
    dcp = cfg.parallel.dcp_size
    pool_tokens = cfg.cache.kv_pool_tokens
    stage_layers = list(range(*pipe.layer_range(cfg.model.num_hidden_layers))) if pipe is not None else None
    if pool_tokens is None and cfg.cache.size_by_memory and device.type == "cuda":
        free, total = torch.cuda.mem_get_info(device)
        pool_tokens = memory_pool_tokens(cfg.model, cfg.cache.gpu_memory_utilization, free, total, ctx, stage_layers, dcp)
        if comm is not None or pipe is not None:
            # every rank (and every stage) runs the same scheduler: they must agree on the pool, so take the smallest
            import torch.distributed as dist
            seen = [None] * dist.get_world_size()
            dist.all_gather_object(seen, pool_tokens)
            pool_tokens = min(seen)
    pools = size_pools(cfg.model, sc.max_num_seqs, ctx, sc.max_num_batched_tokens, dcp, pool_tokens)
    if cfg.cache.num_pages is not None:
        pools["swa_pages"] = max(pools["swa_pages"], cfg.cache.num_pages)
    has_c128 = any(cfg.model.layer_kind(i) == "c128a" for i in range(cfg.model.num_hidden_layers))
    spec_on = cfg.spec.method == "dspark"
    return KVManager(cfg.model, device, sc.max_num_seqs, ctx + 64, pools["swa_pages"] + (sc.max_num_seqs if spec_on else 0),
                     pools["c4_pages"], pools["c128_pages"] if has_c128 else 0, sc.max_num_batched_tokens, layers=stage_layers,
                     extra_swa_layers=cfg.model.n_mtp_layers if spec_on else 0,
                     spec_tokens=cfg.spec.num_speculative_tokens if spec_on else 0, dcp_rank=tp_rank if dcp > 1 else 0,
                     dcp_size=dcp)


def _dsv4_model(cfg: EngineConfig, weights, kv, comm, tp_rank: int):
    from .dsv4 import DSV4Model
    return DSV4Model(cfg.model, weights, kv, comm, tp_rank, cfg.parallel.tp_size)


# ---- layer-by-layer decoders -----------------------------------------------------------------
def _hybrid_shapes(cfg):
    from .hybrid import weight_shapes
    return weight_shapes(cfg)


def _hybrid_weights(cfg, src, device, tp_rank=0, tp_size=1, layer_range=None):
    from .hybrid import build_hybrid_weights
    return build_hybrid_weights(cfg, src, device)


def _hybrid_cache(cfg: EngineConfig, device, ctx: int, comm, tp_rank: int, pipe):
    from ..runtime.kv import HybridKVManager, hybrid_bytes_per_context_token
    sc = cfg.sched
    pool_tokens = cfg.cache.kv_pool_tokens
    per_token = hybrid_bytes_per_context_token(cfg.model)
    if pool_tokens is None and cfg.cache.size_by_memory and device.type == "cuda" and per_token:
        free, total = torch.cuda.mem_get_info(device)
        budget = cfg.cache.gpu_memory_utilization * total - (total - free)
        pool_tokens = max(ctx, int(budget / per_token))
    return HybridKVManager(cfg.model, device, sc.max_num_seqs, ctx + 64, sc.max_num_batched_tokens, cfg.cache.num_pages or 0,
                           pool_tokens)


def _hybrid_model(cfg: EngineConfig, weights, kv, comm, tp_rank: int):
    from .hybrid import HybridModel
    return HybridModel(cfg.model, weights, kv)


_HYBRID_SOURCES = ("elementwise.cu", "meta.cu", "gemm_tcgen05.cu", "skinny.cu", "linear_f32.cu", "hybrid_block.cu", "sampler.cu")
_MECHANISM_SOURCES = {"attention": ("window_attention.cu", "window_attention_tc.cu"), "mlstm": ("mlstm.cu",), "dense": (),
                      "latent_attention": ("latent_attention.cu", "latent_tokens_tc.cu", "latent_prompt_tc.cu"),
                      "grouped_attention": ("window_attention.cu", "latent_prompt_tc.cu", "grouped_attention.cu"),
                      "talking_attention": ("talking_attention.cu", "talking_tokens_tc.cu", "talking_prompt_tc.cu"),
                      "time_mix": ("linear_scan.cu", "retention.cu", "time_mix.cu"), "token_shift": ("token_shift.cu",),
                      "retention": ("linear_scan.cu", "retention.cu"), "mamba2": ("linear_scan.cu", "mamba2.cu"),
                      "moe": ("moe.cu", "moe_plain.cu", "gate_cluster.cu")}


def _hybrid_sources(cfg) -> Tuple[str, Tuple[str, ...]]:
    kinds = [k for k in cfg.mechanisms() if _MECHANISM_SOURCES[k]]
    return "-".join(["hybrid"] + kinds), _HYBRID_SOURCES + tuple(dict.fromkeys(f for k in kinds for f in _MECHANISM_SOURCES[k]))


FAMILIES: Dict[str, ModelFamily] = {
    "dsv4": ModelFamily("dsv4", _dsv4_shapes, _dsv4_weights, _dsv4_cache, _dsv4_model, prefix_cache=True),
    "hybrid": ModelFamily("hybrid", _hybrid_shapes, _hybrid_weights, _hybrid_cache, _hybrid_model, prefix_cache=False,
                          native_sources=_hybrid_sources),
}

# architecture name in config.json -> configuration parser
ARCHITECTURES: Dict[str, Callable[..., Any]] = {
    "Timalorn": timalorn_config_from_json,
    "Domilix": domilix_config_from_json,
    "Fanulix": fanulix_config_from_json,
    "Fogizen": fogizen_config_from_json,
}


def use_native(cfg) -> None:
    """Load the kernels a model needs (compiling them when the checkout has none); before the first kernel of the process."""
    f = family_of(cfg)
    if f.native_sources is not None:
        from ..ops import _lib
        _lib.use_family(*f.native_sources(cfg))


def family_of(cfg) -> ModelFamily:
    return FAMILIES[cfg.family]


def config_from_json(d: Mapping[str, Any], dtype: Optional[str] = None):
    """Configuration object of a `config.json` dictionary.  dtype: compute type for architectures that offer a choice."""
    if not isinstance(d, Mapping):
        raise ConfigError("config.json is not an object")
    arch = d.get("architecture")
    if arch is None and d.get("architectures"):
        arch = d["architectures"][0]
    if isinstance(arch, str) and arch in ARCHITECTURES:
        return ARCHITECTURES[arch](d, dtype or "bfloat16")
    if "architecture" in d:
        raise ConfigError(f"unknown architecture {arch!r} (known: {sorted(ARCHITECTURES)})")
    if dtype == "float32":
        raise ConfigError("this architecture does not run in float32")
    return model_config_from_hf(d)


def load_model_config(path: str, dtype: Optional[str] = None):
    with open(os.path.join(path, "config.json")) as f:
        return config_from_json(json.load(f), dtype)
