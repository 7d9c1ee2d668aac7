"""Registry of the designs that are read from a model folder (`config.json` + `*.safetensors`), and the loader.

`config.json` names its design under "architecture"; the design's module provides `parse_config`, `check_tensors`,
`pack` and `random_tensors`, and registered geometries for random-init runs (`CONFIGS`)."""
from __future__ import annotations

import json
import os
from typing import Dict

from . import kuzanex, ratilorn, tebivik, tuzupel
from .layered_config import LayeredConfig

DESIGNS = {m.ARCHITECTURE: m for m in (kuzanex, tebivik, tuzupel, ratilorn)}
LAYERED_REGISTRY: Dict[str, LayeredConfig] = {name: c for m in DESIGNS.values() for name, c in m.CONFIGS.items()}


class UnknownArchitecture(ValueError):
    pass


def is_model_folder(path: str) -> bool:
    """A folder whose config.json names an architecture (whether or not it is registered)."""
    try:
        with open(os.path.join(path, "config.json"), encoding="utf-8") as f:
            return "architecture" in json.load(f)
    except (OSError, ValueError):
        return False


def read_config(path: str) -> LayeredConfig:
    with open(os.path.join(path, "config.json"), encoding="utf-8") as f:
        c = json.load(f)
    design = DESIGNS.get(c.get("architecture"))
    if design is None:
        raise UnknownArchitecture(f"{path}: architecture {c.get('architecture')!r} is not registered ({', '.join(sorted(DESIGNS))})")
    try:
        return design.parse_config(c, os.path.basename(os.path.abspath(path)) or design.ARCHITECTURE.lower())
    except KeyError as e:
        raise ValueError(f"{path}: config.json has no {e}") from None


def load_folder(path: str, device, dtype=None):
    """(configuration, packed weights) of a model folder, on `device` in the activation type `dtype` (default bf16)."""
    import torch
    from ..convert.safetensors_io import SafetensorsSource
    cfg = read_config(path)
    design = DESIGNS[cfg.architecture]
    src = SafetensorsSource(path)
    try:
        design.check_tensors(cfg, lambda n: src.shape(n) if n in src else None)
        return cfg, design.pack(cfg, src.tensor, dtype or torch.bfloat16, device)
    finally:
        src.close()


def random_layered_weights(cfg: LayeredConfig, device, seed: int = 0, dtype=None) -> dict:
    import torch
    design = DESIGNS[cfg.architecture]
    t = design.random_tensors(cfg, seed, device=device)
    return design.pack(cfg, t.__getitem__, dtype or torch.bfloat16, device)


def save_folder(path: str, cfg: LayeredConfig, tensors: dict) -> None:
    """Writes config.json and model.safetensors (checkpoint tensors, design names)."""
    from ..convert.safetensors_io import write_safetensors
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w", encoding="utf-8") as f:
        json.dump(DESIGNS[cfg.architecture].config_dict(cfg), f, indent=1)
    write_safetensors(os.path.join(path, "model.safetensors"), tensors)
