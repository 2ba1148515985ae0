"""Model designs by the name in their config.json, and the one loader every front end goes through.

A design says how it is loaded and what it is served with: ``"memory"`` (retrieval over a document bank,
``MSAService``) or ``"states"`` (per-sequence state slots, ``scheduler.Scheduler``)."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Any, Callable, Dict

import torch

from .hybrid_config import DESIGNS as HYBRID_DESIGNS


@dataclass(frozen=True)
class Design:
    name: str
    serves: str                                          # "memory" or "states"
    load: Callable[[str, Any, torch.dtype], Any]         # (path, device, dtype) -> model
    dtypes: tuple = (torch.bfloat16,)


_DESIGNS: Dict[str, Design] = {}


def register(design: Design) -> None:
    _DESIGNS[design.name] = design


def designs() -> Dict[str, Design]:
    return dict(_DESIGNS)


def design_of(path: str) -> Design:
    """The design of the checkpoint in ``path``: its config.json's ``architecture`` or first ``architectures`` entry; a
    configuration with an ``msa_config`` is the memory model whatever its class is called."""
    with open(os.path.join(path, "config.json")) as f:
        raw = json.load(f)
    name = raw.get("architecture") or (raw.get("architectures") or [""])[0]
    if name in _DESIGNS:
        return _DESIGNS[name]
    if "msa_config" in raw or raw.get("model_type") == "msa":
        return _DESIGNS["MSAForCausalLM"]
    raise ValueError(f"{path}: unknown architecture {name!r} (known: {sorted(_DESIGNS)})")


def load_model(path: str, device, dtype: torch.dtype = torch.bfloat16):
    design = design_of(path)
    if dtype not in design.dtypes:
        raise ValueError(f"{design.name} runs in {design.dtypes}, not {dtype}")
    return design.load(path, device, dtype)


def _load_msa(path, device, dtype):
    from .prefill import load_msa_checkpoint
    return load_msa_checkpoint(path, device, dtype)


def _load_hybrid(path, device, dtype):
    from .hybrid import HybridForCausalLM
    return HybridForCausalLM.from_pretrained(path, device, dtype)


register(Design("MSAForCausalLM", "memory", _load_msa, (torch.bfloat16, torch.float32)))
for _name in HYBRID_DESIGNS:
    register(Design(_name, "states", _load_hybrid, (torch.bfloat16, torch.float32)))
