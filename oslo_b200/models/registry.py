"""Which classes a ``config.json`` belongs to.

A configuration names its model by ``model_type`` (``"gptj"``), by ``architectures`` (``["GPTJForCausalLM"]``) or by
``architecture`` (``"Moronex"``). ``load_causal_lm(directory)`` reads it, picks the classes and loads the weights.
"""
from __future__ import annotations

import json
import os
from typing import Any, Dict, NamedTuple, Type

from ..modeling_utils import CONFIG_NAME, PretrainedConfig, PreTrainedModel, _resolve_hub_file
from .begovik import BegovikConfig, BegovikForCausalLM
from .dekutar import DekutarConfig, DekutarForCausalLM
from .gpt2 import GPT2Config, GPT2LMHeadModel
from .gpt_neo import GPTNeoConfig, GPTNeoForCausalLM
from .gptj import GPTJConfig, GPTJForCausalLM
from .masezen import MasezenConfig, MasezenForCausalLM
from .moronex import MoronexConfig, MoronexForCausalLM


class ModelEntry(NamedTuple):
    config: Type[PretrainedConfig]
    causal_lm: Type[PreTrainedModel]


MODELS: Dict[str, ModelEntry] = {
    "gpt2": ModelEntry(GPT2Config, GPT2LMHeadModel),
    "gpt_neo": ModelEntry(GPTNeoConfig, GPTNeoForCausalLM),
    "gptj": ModelEntry(GPTJConfig, GPTJForCausalLM),
    "moronex": ModelEntry(MoronexConfig, MoronexForCausalLM),
    "begovik": ModelEntry(BegovikConfig, BegovikForCausalLM),
    "dekutar": ModelEntry(DekutarConfig, DekutarForCausalLM),
    "masezen": ModelEntry(MasezenConfig, MasezenForCausalLM),
}


def find_model(config: Dict[str, Any]) -> ModelEntry:
    """The entry of a parsed ``config.json``."""
    kind = config.get("model_type")
    if kind in MODELS:
        return MODELS[kind]
    names = [str(n) for n in ([config.get("architecture")] + list(config.get("architectures") or [])) if n]
    for name in names:
        for key, entry in MODELS.items():
            if name.lower() == key or name == entry.causal_lm.__name__:
                return entry
    raise ValueError(f"no model for model_type {kind!r} / architectures {names}; known: {sorted(MODELS)}")


def load_causal_lm(name_or_path: str, **kwargs: Any) -> PreTrainedModel:
    """``from_pretrained`` of whichever causal-LM class the checkpoint's ``config.json`` names."""
    path = os.path.join(name_or_path, CONFIG_NAME) if os.path.isdir(name_or_path) else _resolve_hub_file(name_or_path, CONFIG_NAME)
    with open(path, "r", encoding="utf-8") as f:
        raw = json.load(f)
    entry = find_model(raw)
    return entry.causal_lm.from_pretrained(name_or_path, **kwargs)
