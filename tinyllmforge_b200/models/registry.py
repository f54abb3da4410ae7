"""Model registry: from a ``config.json`` to its configuration class and its model class.

An entry names the configuration class (a dataclass with ``from_dict``) and the model class.  A checkpoint of
Goselix, Tonapel, Mezapel or Galupel names its design under ``architecture``; everything else is a Hugging Face configuration whose
``model_type`` the configuration class checks itself.
"""
from __future__ import annotations

import importlib
import json
import os

# name -> (configuration class, model class), imported on first use
_ENTRIES = {
    "qwen3": ("tinyllmforge_b200.config:ModelConfig", "tinyllmforge_b200.models.qwen3:Qwen3ForCausalLM"),
    "Goselix": ("tinyllmforge_b200.models.goselix_config:GoselixConfig", "tinyllmforge_b200.models.goselix:GoselixForCausalLM"),
    "Tonapel": ("tinyllmforge_b200.models.tonapel_config:TonapelConfig", "tinyllmforge_b200.models.tonapel:TonapelForCausalLM"),
    "Mezapel": ("tinyllmforge_b200.models.mezapel_config:MezapelConfig", "tinyllmforge_b200.models.mezapel:MezapelForCausalLM"),
    "Galupel": ("tinyllmforge_b200.models.galupel_config:GalupelConfig", "tinyllmforge_b200.models.galupel:GalupelForCausalLM"),
}


def _resolve(path: str):
    module, name = path.split(":")
    return getattr(importlib.import_module(module), name)


def architectures() -> list[str]:
    return sorted(_ENTRIES)


def config_from_dict(d: dict):
    name = d.get("architecture") or "qwen3"
    if name not in _ENTRIES:
        raise ValueError(f"unknown architecture {name!r}; known: {architectures()}")
    return _resolve(_ENTRIES[name][0]).from_dict(d)


def config_from_dir(path: str):
    with open(os.path.join(path, "config.json")) as f:
        return config_from_dict(json.load(f))


def model_class(cfg):
    for config_path, model_path in _ENTRIES.values():
        if type(cfg) is _resolve(config_path):
            return _resolve(model_path)
    raise ValueError(f"no model class is registered for {type(cfg).__name__}")
