"""Which models the engine serves: how a family is recognised, how its weights are read and which engine class runs it.

A model on disk is either one file (a GPT-2 archive, ``.nxs`` or ``.pt``) or a folder with ``config.json``, whose
``architecture`` names the family.  :func:`load_model` reads either, :func:`create_engine` picks the engine class from the
weights, :func:`open_engine` does both."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, Dict, Optional

from ..lm.gutivik import load_gutivik
from ..lm.hybrid import HybridWeights, load_gugedra
from ..lm.lukopel import load_lukopel
from ..lm.makuzen import load_makuzen
from .engine import Engine, EngineConfig, Gpt2Weights, load_gpt2
from .hybrid import HybridEngine

__all__ = ["ModelFamily", "register_family", "families", "load_model", "create_engine", "open_engine"]


@dataclass(frozen=True)
class ModelFamily:
    name: str                            # the `architecture` of config.json
    load: Callable[[str], object]        # path -> weights
    weights: type                        # what `load` returns
    engine: type                         # the Engine class that runs these weights


_FAMILIES: Dict[str, ModelFamily] = {}


def register_family(family: ModelFamily) -> None:
    if family.name in _FAMILIES:
        raise ValueError(f"model family {family.name!r} is registered already")
    _FAMILIES[family.name] = family


def families() -> Dict[str, ModelFamily]:
    return dict(_FAMILIES)


def load_model(path: str):
    """Weights of a model file or folder."""
    if not os.path.isdir(path):
        return _FAMILIES["GPT2"].load(path)
    with open(os.path.join(path, "config.json")) as f:
        name = json.load(f).get("architecture")
    if name not in _FAMILIES:
        raise ValueError(f"unknown architecture {name!r} (known: {', '.join(sorted(_FAMILIES))})")
    return _FAMILIES[name].load(path)


def create_engine(weights, config: Optional[EngineConfig] = None, group=None) -> Engine:
    for f in _FAMILIES.values():
        if isinstance(weights, f.weights):
            return f.engine(weights, config, group)
    raise TypeError(f"no model family serves {type(weights).__name__}")


def open_engine(path: str, config: Optional[EngineConfig] = None, group=None) -> Engine:
    return create_engine(load_model(path), config, group)


def _load_gpt2_folder(path: str) -> Gpt2Weights:
    return load_gpt2(os.path.join(path, "model.nxs") if os.path.isdir(path) else path)


register_family(ModelFamily("GPT2", _load_gpt2_folder, Gpt2Weights, Engine))
register_family(ModelFamily("Gugedra", load_gugedra, HybridWeights, HybridEngine))
register_family(ModelFamily("Makuzen", load_makuzen, HybridWeights, HybridEngine))
register_family(ModelFamily("Gutivik", load_gutivik, HybridWeights, HybridEngine))
register_family(ModelFamily("Lukopel", load_lukopel, HybridWeights, HybridEngine))
