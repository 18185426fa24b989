"""Model families by architecture name: how a ``config.json`` becomes a model configuration, where weights come
from, and which engine runs them. Everything that starts from a configuration (``config.parse_config``, the
serving command line, the trace replay) goes through here.
"""
from __future__ import annotations

import os
from dataclasses import dataclass
from typing import Any, Callable, Dict


@dataclass(frozen=True)
class ModelFamily:
    name: str
    architectures: tuple
    parse_model: Callable[..., Any]          # (config.json dict, tp=, run_layers=, name=) -> model configuration
    load_folder: Callable[..., Any]          # (NanoflowConfig, folder, device) -> weights of a checkpoint folder
    random_weights: Callable[..., Any]       # (NanoflowConfig, rank, tp, device, seed) -> weights
    engine: Callable[..., Any]               # (NanoflowConfig, weights, **kw) -> engine
    cpu_engine: Callable[..., Any]           # (NanoflowConfig, list of per-rank weights, num_pages=) -> CPU engine
    complete: Callable[..., Any] = None      # (config.json dict, checkpoint folder) -> the dict with sizes from the tensors
    listed_layers: bool = False              # the layers are listed one by one in config.json
    runs_float32: bool = False               # the engine can store and multiply in 32-bit


def _llama() -> ModelFamily:
    from ..config import ModelConfig
    from .llama import random_rank_weights, shard_weights

    def load_folder(cfg, folder, device):
        from .weights import load_hf_checkpoint
        return shard_weights(load_hf_checkpoint(folder), cfg.model, 0, 1, device=device)

    def random(cfg, rank, tp, device, seed=0):
        return random_rank_weights(cfg.model, rank, tp, device, seed=seed, o1=bool(cfg.engine.o_allgather_nanos))

    def engine(cfg, weights, **kw):
        from ..runtime.engine import Engine
        return Engine(cfg, weights, **kw)

    def cpu_engine(cfg, shards, num_pages=256):
        from ..runtime.cpu_backend import CpuEngine
        return CpuEngine(cfg, shards, num_pages=num_pages)

    return ModelFamily("llama", ("LlamaForCausalLM", "Qwen2ForCausalLM", "MixtralForCausalLM"), ModelConfig.from_hf,
                       load_folder, random, engine, cpu_engine)


def _layer_list(name: str, design) -> ModelFamily:
    """Family of a layer-list design: a module of ``models/`` with its keys, tensor names and random weights."""

    def load_folder(cfg, folder, device):
        return design.load_weights(cfg.model, folder, device)

    def random(cfg, rank, tp, device, seed=0):
        return design.random_weights(cfg.model, cfg.raw["model"], device, seed)

    def engine(cfg, weights, **kw):
        from ..runtime.layer_list import LayerListEngine
        return LayerListEngine(cfg, weights, **kw)

    def cpu_engine(cfg, shards, num_pages=256):
        from ..runtime.cpu_layer_list import CpuLayerListEngine
        return CpuLayerListEngine(cfg, shards[0], num_pages=num_pages)

    return ModelFamily(name, (design.ARCHITECTURE,), design.parse_model, load_folder, random, engine, cpu_engine,
                       complete=getattr(design, "complete", None), listed_layers=True, runs_float32=True)


def _volarax() -> ModelFamily:
    from . import volarax
    return _layer_list("volarax", volarax)


def _zubedra() -> ModelFamily:
    from . import zubedra
    return _layer_list("zubedra", zubedra)


def _gupizen() -> ModelFamily:
    from . import gupizen
    return _layer_list("gupizen", gupizen)


def _gimudra() -> ModelFamily:
    from . import gimudra
    return _layer_list("gimudra", gimudra)


_FAMILIES: Dict[str, Callable[[], ModelFamily]] = {"llama": _llama, "volarax": _volarax, "zubedra": _zubedra,
                                                    "gupizen": _gupizen, "gimudra": _gimudra}
_cache: Dict[str, ModelFamily] = {}


def family(name: str) -> ModelFamily:
    if name not in _cache:
        _cache[name] = _FAMILIES[name]()
    return _cache[name]


def architecture_of(hf: Dict[str, Any]) -> str:
    return hf.get("architecture") or (hf.get("architectures") or [""])[0]


def family_of(hf: Dict[str, Any]) -> ModelFamily:
    """Family of a ``config.json`` dictionary. One that names no architecture is taken for a Llama, as ever;
    one that names an unknown architecture is taken for a Llama if it has a Llama's keys."""
    arch = architecture_of(hf)
    for name in _FAMILIES:
        if arch in family(name).architectures:
            return family(name)
    if "num_attention_heads" in hf:
        return family("llama")
    raise ValueError(f"unknown architecture '{arch}' (known: "
                     f"{', '.join(a for n in _FAMILIES for a in family(n).architectures)})")


def is_model_folder(path: str) -> bool:
    return bool(path) and os.path.isfile(os.path.join(path, "config.json")) and \
        any(f.endswith(".safetensors") for f in os.listdir(path))
