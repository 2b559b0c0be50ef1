"""Architectures that are read from their own checkpoint format: `config.json` with an "architecture" key next to one
`model.safetensors`.  An entry is a module with

    read_config(dict) -> ModelConfig          load_weights(directory, cfg, device, dtype) -> W
    random_weights(cfg, device, seed, dtype) -> W

Everything behind the nested weight dict W (runner, caches, scheduler, server) is shared by all families."""
from __future__ import annotations

import importlib

ARCHITECTURES = {"Vabunex": "vabunex", "Debisun": "debisun", "Zapolorn": "zapolorn", "Zakusun": "zakusun"}
FAMILIES = {"vabunex": "vabunex", "debisun": "debisun", "zapolorn": "zapolorn", "zakusun": "zakusun"}


def architecture(d: dict):
    name = d.get("architecture")
    if name not in ARCHITECTURES:
        raise ValueError(f"unknown architecture {name!r} (known: {', '.join(sorted(ARCHITECTURES))})")
    return importlib.import_module("." + ARCHITECTURES[name], __package__)


def family(cfg):
    """The module of a configuration's family, or None for families whose weights come in the serving layout."""
    name = FAMILIES.get(cfg.family)
    return importlib.import_module("." + name, __package__) if name else None
