"""Model families by the architecture name of a model folder's config.json."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, Dict, Tuple

import torch

from . import safetensors
from .config import HybridConfig, ModelConfig, sabipel_config


@dataclass(frozen=True)
class ModelFamily:
    architecture: str
    libraries: Tuple[str, ...]                    # the CUDA libraries of its operators (see build.LIBRARIES)
    dtypes: Tuple[torch.dtype, ...]               # activation types it runs in, the default first
    config_from_dict: Callable
    build: Callable                               # (cfg, tensors, dtype, device) -> model

    def build_libraries(self) -> None:
        """Compile what is out of date of the libraries this family needs, and of no other."""
        from ..build import build
        for name in self.libraries:
            build(library=name)


_FAMILIES: Dict[str, ModelFamily] = {}


def register(family: ModelFamily) -> ModelFamily:
    if family.architecture in _FAMILIES:
        raise ValueError(f"{family.architecture} is registered already")
    _FAMILIES[family.architecture] = family
    return family


def architectures():
    return sorted(_FAMILIES)


def family_of(config: dict) -> ModelFamily:
    name = config.get("architecture")
    if name not in _FAMILIES:
        raise ValueError(f"unknown architecture {name!r}; known: {architectures()}")
    return _FAMILIES[name]


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def load_model(folder: str, dtype: torch.dtype = None, device="cuda", config: dict = None):
    """The model of a folder with config.json and model.safetensors, ready for `GenerationRunner`."""
    raw = config if config is not None else read_config(folder)
    family = family_of(raw)
    dtype = dtype or family.dtypes[0]
    if dtype not in family.dtypes:
        raise ValueError(f"{family.architecture} runs in {family.dtypes}, not in {dtype}")
    cfg = family.config_from_dict(raw)
    return family.build(cfg, safetensors.load_file(os.path.join(folder, "model.safetensors")), dtype, device)


def _build_qwen3(cfg, tensors, dtype, device):
    from .model import TPDecoder
    from .weights import rank_weights_from_tensors
    return TPDecoder(cfg, rank_weights_from_tensors(cfg, tensors, 0, 1, device), device=device)


def _build_hybrid(cfg, tensors, dtype, device):
    from .hybrid import HybridDecoder
    from .weights import hybrid_weights
    return HybridDecoder(cfg, hybrid_weights(cfg, tensors, dtype, device), device=device)


register(ModelFamily("Qwen3", ("attention",), (torch.bfloat16,), ModelConfig.from_dict, _build_qwen3))
register(ModelFamily("Berilix", ("rows", "hybrid"), (torch.bfloat16, torch.float32), HybridConfig.from_dict, _build_hybrid))
register(ModelFamily("Sabipel", ("rows", "mixers"), (torch.bfloat16, torch.float32), sabipel_config, _build_hybrid))
