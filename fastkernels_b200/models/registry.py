"""Which model class serves a configuration, and which configuration a folder holds."""
from __future__ import annotations

import importlib
import json
from pathlib import Path

import torch

from .weights import SafetensorsSource, TensorSource

# architecture name in config.json -> module with
#   config_from_json(dict, source, dtype) -> config and MODEL_CLASSES {config type: class}
_ARCHITECTURES = {
    "Pinuvik": "fastkernels_b200.models.pinuvik",
    "Rivilix": "fastkernels_b200.models.rivilix",
    "LlamaForCausalLM": "fastkernels_b200.models.llama",
    "Qwen3ForCausalLM": "fastkernels_b200.models.llama",
}

# parts of the CUDA library (build.COMPONENT_SOURCES) that a module's models call
_LIBRARY_PARTS = {
    "fastkernels_b200.models.llama": ["decode_attn"],
    "fastkernels_b200.models.pinuvik": ["decode_attn", "delta"],
    "fastkernels_b200.models.rivilix": ["latent", "mlstm", "experts"],
}


def architectures() -> list[str]:
    return sorted(_ARCHITECTURES)


def _module_name(name: str) -> str:
    if name not in _ARCHITECTURES:
        raise ValueError(f"unknown architecture '{name}' (known: {', '.join(architectures())})")
    return _ARCHITECTURES[name]


def _module(name: str):
    return importlib.import_module(_module_name(name))


def library_parts(folder) -> list[str]:
    """Parts of the CUDA library that the model in a folder needs beside the core."""
    cfg = json.loads((Path(folder) / "config.json").read_text())
    return _LIBRARY_PARTS[_module_name(architecture_of(cfg))]


def model_class(config):
    """The ServedModel class for a configuration object."""
    for mod_name in dict.fromkeys(_ARCHITECTURES.values()):
        classes = importlib.import_module(mod_name).MODEL_CLASSES
        for config_type, cls in classes.items():
            if isinstance(config, config_type):
                return cls
    raise TypeError(f"no model is registered for {type(config).__name__}")


def architecture_of(cfg: dict) -> str:
    name = cfg.get("architecture") or (cfg.get("architectures") or [None])[0]
    if name is None:
        raise ValueError("config.json names no architecture")
    return name


def load_folder(folder, dtype=torch.bfloat16) -> tuple[object, TensorSource]:
    """(configuration, weights) of a model folder with config.json and safetensors."""
    folder = Path(folder)
    cfg = json.loads((folder / "config.json").read_text())
    source = SafetensorsSource(folder)
    return _module(architecture_of(cfg)).config_from_json(cfg, source, dtype), source
