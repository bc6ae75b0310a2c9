"""Model registry: which engine serves a model folder, by the `architecture` of its config.json."""
from __future__ import annotations

from dataclasses import dataclass, fields
from pathlib import Path
from typing import Any, Callable

import torch

from . import checkpoint


@dataclass(frozen=True)
class Family:
    name: str
    config: Callable                 # config.json dictionary -> configuration object
    load: Callable | None            # (configuration, tensors, dtype, device) -> weights; None: no checkpoint reader
    random: Callable                 # (configuration, seed, dtype, device) -> weights
    engine: Callable                 # (configuration, weights, batch, max_context, device, **options) -> SlotEngine
    dtypes: tuple
    part: str | None = None          # the library part its kernels live in (build.py); None: the whole library


@dataclass
class Model:
    family: Family
    cfg: Any
    weights: Any

    def engine(self, batch: int, max_context: int, device="cuda", **options):
        return self.family.engine(self.cfg, self.weights, batch, max_context, device, **options)


_FAMILIES: dict[str, Family] = {}


def register(family: Family) -> None:
    _FAMILIES[family.name] = family


def families() -> list[str]:
    return sorted(_FAMILIES)


def family(config: dict) -> Family:
    name = config.get("architecture")
    if name not in _FAMILIES:
        raise ValueError(f"unknown architecture {name!r} (known: {', '.join(families())})")
    return _FAMILIES[name]


def _checked(fam: Family, dtype) -> None:
    if dtype not in fam.dtypes:
        raise ValueError(f"{fam.name} does not run in {dtype}")


def load_model(folder, dtype=torch.bfloat16, device="cuda") -> Model:
    config = checkpoint.read_config(folder)
    fam = family(config)
    _checked(fam, dtype)
    if fam.load is None:
        raise ValueError(f"{fam.name} has no checkpoint reader")
    cfg = fam.config(config)
    tensors = checkpoint.read_safetensors(Path(folder) / "model.safetensors")
    return Model(fam, cfg, fam.load(cfg, tensors, dtype, device))


def random_model(config: dict, seed: int = 0, dtype=torch.bfloat16, device="cuda") -> Model:
    fam = family(config)
    _checked(fam, dtype)
    cfg = fam.config(config)
    return Model(fam, cfg, fam.random(cfg, seed, dtype, device))


# ------------------------------------------------------------------------------------------------------------ families
def _hybrid_load(cfg, tensors, dtype, device):
    from .hybrid import HybridWeights
    return HybridWeights(cfg).load(tensors, dtype, device)


def _hybrid_random(cfg, seed, dtype, device):
    from .hybrid import HybridWeights, random_tensors
    weights = HybridWeights(cfg)
    return weights.load(random_tensors(weights, seed, device), dtype, device)


def _hybrid_engine(cfg, weights, batch, max_context, device, **options):
    from .hybrid import HybridEngine
    return HybridEngine(weights, batch, max_context, device, **options)


def _hybrid_config(config):
    from .hybrid import HybridConfig
    return HybridConfig.from_config(config)


def _qwen_config(config):
    from .engine import ModelConfig
    known = {f.name for f in fields(ModelConfig)}
    return ModelConfig(**{k: v for k, v in config.items() if k in known})


def _qwen_random(cfg, seed, dtype, device):
    from .engine import random_weights
    return random_weights(cfg, seed, device)


def _qwen_engine(cfg, weights, batch, max_context, device, **options):
    from .engine import Engine
    return Engine(cfg, weights, batch, max_context, device, **options)


for _name in ("Tofilorn", "Dugilorn"):
    register(Family(_name, _hybrid_config, _hybrid_load, _hybrid_random, _hybrid_engine, (torch.bfloat16, torch.float32), part="hybrid"))
register(Family("Qwen3.5", _qwen_config, None, _qwen_random, _qwen_engine, (torch.bfloat16,)))
