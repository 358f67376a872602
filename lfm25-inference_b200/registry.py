"""Model registry: which family serves a model folder, chosen by the `architecture` of its config.json.

A family is a loader `(folder, config, device, num_pages, num_request_slots, dtype) -> model`; every model offers
`create_engine` (the serving engine's hook), `vocab`, `num_pages` and `num_request_slots`.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable

from . import fegidra, ribivik


class UnknownModel(ValueError):
    pass


class UnsupportedType(ValueError):
    """The family has no kernels for the asked activation type."""


@dataclass(frozen=True)
class Family:
    architecture: str
    load: Callable
    dtypes: tuple[str, ...]


def _load_lfm2_random(folder: str, config: dict, device, num_pages: int, num_request_slots: int, dtype: str):
    """LFM2.5-1.2B shapes with weights drawn from `seed` (no checkpoint of it is part of this repository)."""
    from .model import RandomModel
    return RandomModel(int(config.get("seed", 0)), device, num_pages, num_request_slots,
                       fp8_policy=bool(config.get("fp8", False)))


FAMILIES = {family.architecture: family for family in (
    Family(fegidra.ARCHITECTURE, fegidra.load, ("bfloat16", "float32")),
    Family(ribivik.ARCHITECTURE, ribivik.load, ("bfloat16", "float32")),
    Family("Lfm2Random", _load_lfm2_random, ("bfloat16",)),
)}


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as handle:
        return json.load(handle)


def family_of(config: dict) -> Family:
    name = config.get("architecture")
    if name not in FAMILIES:
        raise UnknownModel(f"no model family for architecture {name!r}; known: {', '.join(sorted(FAMILIES))}")
    return FAMILIES[name]


def load_model(folder: str, device, num_pages: int, num_request_slots: int, dtype: str = "bfloat16"):
    config = read_config(folder)
    family = family_of(config)
    if dtype not in family.dtypes:
        raise UnsupportedType(f"{family.architecture} runs in {', '.join(family.dtypes)}, not {dtype}")
    return family.load(folder, config, device, num_pages, num_request_slots, dtype)
