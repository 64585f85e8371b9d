"""Base models by the architecture a checkpoint's config.json names."""
import json
import os
from typing import Any, Dict, List

import torch

from . import modeling_dilavik, modeling_llama, modeling_nulunex

# architecture name -> class with from_pretrained(path, torch_dtype, device)
_MODELS: Dict[str, Any] = {}


def register(name: str, model_class) -> None:
    _MODELS[name] = model_class


def architectures() -> List[str]:
    return sorted(_MODELS)


def architecture_of(config: Dict[str, Any]) -> str:
    """'architecture', or the first of 'architectures', or the model type (Hugging Face directories)."""
    name = config.get("architecture")
    if name is None and config.get("architectures"):
        name = config["architectures"][0]
    if name is None and config.get("model_type") == "llama":
        name = "LlamaForCausalLM"
    if name not in _MODELS:
        raise ValueError(f"unknown architecture {name!r}: this framework has {', '.join(architectures())}")
    return name


def model_class_of(path: str):
    with open(os.path.join(path, "config.json")) as f:
        return _MODELS[architecture_of(json.load(f))]


def load_model(path: str, torch_dtype: torch.dtype = torch.bfloat16, device="cuda"):
    """The base model of a checkpoint directory."""
    return model_class_of(path).from_pretrained(path, torch_dtype=torch_dtype, device=device)


def new_model(config: Dict[str, Any], torch_dtype: torch.dtype = torch.bfloat16, device="cuda"):
    """A base model without weights, from the contents of a nested config.json (the classes that name their config_class)."""
    cls = _MODELS[architecture_of(config)]
    with torch.device(device):
        return cls(cls.config_class.from_dict(config)).to(torch_dtype)


register("LlamaForCausalLM", modeling_llama.LlamaForCausalLM)
register("Dilavik", modeling_dilavik.DilavikForCausalLM)
register("Nulunex", modeling_nulunex.NulunexForCausalLM)
