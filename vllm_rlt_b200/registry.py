"""The model registry: an architecture name from config.json to a configuration and a model class.

A model class is constructed as `model_class(config, state_dict, device, dtype)` and serves through the engine
with four methods:

    model.cache_spec()                -> CacheSpec: what a sequence keeps in pages and in its state slot
    model.forward_step(batch, cache)  -> opaque hidden state of all rows of a step
    model.step_logits(hidden, rows)   -> fp32 logits of the given rows (None: all of them)
    model.vocab_size
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Callable

import torch

from .checkpoint import read_config, read_weights
from .hybrid_lm import HybridLM, HybridLMConfig
from .looped_lm import LoopedLM, LoopedLMConfig
from .postnorm_lm import PostNormLM, PostNormLMConfig
from .sandwich_lm import SandwichLM, SandwichLMConfig
from .stream_lm import StreamLM, StreamLMConfig


@dataclass(frozen=True)
class ModelFamily:
    architecture: str
    parse_config: Callable[[dict], object]
    model_class: type


_FAMILIES: dict[str, ModelFamily] = {}


def register_model(architecture: str, parse_config, model_class) -> None:
    if architecture in _FAMILIES:
        raise ValueError(f"architecture {architecture} is already registered")
    _FAMILIES[architecture] = ModelFamily(architecture, parse_config, model_class)


def registered_architectures() -> list[str]:
    return sorted(_FAMILIES)


def resolve(config: dict) -> ModelFamily:
    """The family a config.json names (`architecture`, or the first of `architectures`)."""
    name = config.get("architecture") or next(iter(config.get("architectures") or []), None)
    family = _FAMILIES.get(name)
    if family is None:
        raise ValueError(f"unknown architecture {name!r}; registered: {', '.join(registered_architectures())}")
    return family


def load_model(folder, *, device="cuda", dtype: torch.dtype = torch.bfloat16):
    """The model of a folder with config.json and safetensors weights."""
    config = read_config(folder)
    family = resolve(config)
    return family.model_class(family.parse_config(config), read_weights(folder), device, dtype)


register_model("OuroForCausalLM", LoopedLMConfig.from_json, LoopedLM)
register_model("Sobipel", HybridLMConfig.from_json, HybridLM)
register_model("Sugosun", StreamLMConfig.from_json, StreamLM)
register_model("Kezuvik", SandwichLMConfig.from_json, SandwichLM)
register_model("Degavik", PostNormLMConfig.from_json, PostNormLM)
