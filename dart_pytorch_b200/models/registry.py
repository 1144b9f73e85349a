"""Which model family a ``config.json`` describes, and how families that are built from it are constructed.

Families of the Hugging Face loaders are named by ``model_type``; others by ``architecture``.  ``apps.servers.load_hf_model``
resolves the family ``"auto"`` through this table, so every runner and service takes any of them.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, Dict

HF_MODEL_TYPES = {"gpt2": "gpt2", "gpt_neox": "pythia", "gptj": "gptj", "llama": "llama"}


@dataclass(frozen=True)
class Architecture:
    """A family whose sizes and constants all come from ``config.json`` and the checkpoint's shapes."""
    family: str
    build: Callable            # (config dict, checkpoint or None, **kw) -> model
    load_map: Callable         # (model, state dict) -> LoadReport


def _famudra() -> Architecture:
    from ..io.famudra_loader import FamudraLoader
    from .famudra import Famudra, FamudraConfig
    return Architecture("famudra", lambda config, state=None, **kw: Famudra(FamudraConfig.from_json(config, **kw)),
                        FamudraLoader.load_map)


def _pozalorn() -> Architecture:
    from ..io.pozalorn_loader import PozalornLoader
    from .pozalorn import Pozalorn, PozalornConfig
    return Architecture("pozalorn", lambda config, state=None, **kw: Pozalorn(PozalornConfig.from_json(config, state, **kw)),
                        PozalornLoader.load_map)


ARCHITECTURES: Dict[str, Callable[[], Architecture]] = {"famudra": _famudra, "pozalorn": _pozalorn}


def read_config(model_dir: str) -> dict:
    with open(os.path.join(model_dir, "config.json"), "r", encoding="utf-8") as f:
        return json.load(f)


def family_of(config: dict) -> str:
    name = str(config.get("architecture", "")).lower()
    if name in ARCHITECTURES:
        return name
    kind = str(config.get("model_type", "")).lower()
    if kind in HF_MODEL_TYPES:
        return HF_MODEL_TYPES[kind]
    raise ValueError(f"config.json names no known model family (architecture {config.get('architecture')!r}, "
                     f"model_type {config.get('model_type')!r})")


def architecture(family: str) -> Architecture:
    return ARCHITECTURES[family]()
