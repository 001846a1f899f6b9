"""Model designs by name.

A checkpoint folder holds ``config.json`` and ``model.safetensors``; ``config.json`` names its design
under ``architecture``. A design registers how its configuration is read and which model class holds
its weights; the inference engine picks the matching engine class from the configuration's type.
``.oil`` files keep carrying their own configuration and do not go through this table.
"""
from __future__ import annotations

import importlib
import json
import os
from dataclasses import dataclass
from typing import Callable


@dataclass(frozen=True)
class Architecture:
    name: str
    config_from_dict: Callable[[dict], object]
    model: str                       # "module:Class" (imported on first use)

    def model_class(self):
        mod, cls = self.model.split(":")
        return getattr(importlib.import_module(mod), cls)


ARCHITECTURES: dict[str, Architecture] = {}


def register(name: str, config_from_dict, model: str) -> None:
    ARCHITECTURES[name] = Architecture(name, config_from_dict, model)


def architecture(name: str) -> Architecture:
    from . import hybrid_config  # noqa: F401 - registers the designs of this package

    if name not in ARCHITECTURES:
        raise KeyError(f"unknown model design {name!r}; known: {', '.join(sorted(ARCHITECTURES))}")
    return ARCHITECTURES[name]


def is_checkpoint_dir(path: str) -> bool:
    return os.path.isdir(path) and os.path.exists(os.path.join(path, "config.json"))


def load_config(path: str):
    """``(architecture, config)`` of a checkpoint folder."""
    with open(os.path.join(path, "config.json"), encoding="utf-8") as f:
        raw = json.load(f)
    arch = architecture(str(raw.get("architecture", "")))
    return arch, arch.config_from_dict(raw)


def load_checkpoint(path: str, device="cpu"):
    """Model of a checkpoint folder, weights in their stored types on ``device``."""
    from ..oil.importers import read_safetensors_torch

    arch, cfg = load_config(path)
    tensors = read_safetensors_torch(os.path.join(path, "model.safetensors"))
    return arch.model_class()(cfg, tensors).to(device)
