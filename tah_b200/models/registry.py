"""Model families by what ``config.json`` says: how to load a checkpoint directory and which engine serves the model.

``load_model(path)`` and ``make_engine(model)`` are what the command lines, the evaluation backends and the trace replay
use, so a further family only registers itself here.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, List, Optional

import torch


@dataclass(frozen=True)
class Family:
    name: str
    matches: Callable[[dict], bool]               # config.json -> is it this family?
    load: Callable[..., object]                   # (path, dtype, device) -> model
    owns: Callable[[object], bool]                # model instance -> is it this family?
    engine: Callable[..., object]                 # (model, **engine options) -> engine
    sources: Optional[str] = None                 # kernel source group that suffices to serve it, None = all


_FAMILIES: List[Family] = []


def register_family(family: Family) -> None:
    _FAMILIES[:] = [f for f in _FAMILIES if f.name != family.name] + [family]


def families() -> List[str]:
    return [f.name for f in _FAMILIES]


def read_config(path: str) -> dict:
    with open(os.path.join(path, "config.json"), encoding="utf-8") as fh:
        return json.load(fh)


def family_of_config(config: dict) -> Family:
    for f in _FAMILIES:
        if f.matches(config):
            return f
    arch = config.get("architecture") or config.get("architectures") or config.get("model_type")
    raise ValueError(f"no model family for architecture {arch!r}; have {families()}")


def family_of_model(model) -> Family:
    for f in _FAMILIES:
        if f.owns(model):
            return f
    raise TypeError(f"no model family for {type(model).__name__}; have {families()}")


def load_model(path: str, dtype: torch.dtype = None, device=None):
    """Load a checkpoint directory of any registered family."""
    return family_of_config(read_config(path)).load(path, dtype, device)


def make_engine(model, **kw):
    """A new engine for ``model`` (see the family's engine class for the options)."""
    return family_of_model(model).engine(model, **kw)


# ------------------------------------------------------------------------------------
# built-in families (imports stay inside: loading one family does not import the others)
# ------------------------------------------------------------------------------------
def _qwen3_matches(c: dict) -> bool:
    return c.get("model_type") == "qwen3" or "Qwen3ForCausalLM" in (c.get("architectures") or [])


def _qwen3_load(path, dtype, device):
    from tah_b200.model.tah_model import TaHForCausalLM
    return TaHForCausalLM.from_pretrained(path, torch_dtype=dtype, device=device)


def _qwen3_owns(model) -> bool:
    return hasattr(model, "simple_base_model")


def _qwen3_engine(model, **kw):
    from tah_b200.engine.engine import TaHEngine
    return TaHEngine(model, **kw)


def _gunuvik_load(path, dtype, device):
    from tah_b200.models.gunuvik import GunuvikForCausalLM
    return GunuvikForCausalLM.from_pretrained(path, dtype=dtype, device=device)


def _ditilix_load(path, dtype, device):
    from tah_b200.models.ditilix import DitilixForCausalLM
    return DitilixForCausalLM.from_pretrained(path, dtype=dtype, device=device)


def _niralix_load(path, dtype, device):
    from tah_b200.models.niralix import NiralixForCausalLM
    return NiralixForCausalLM.from_pretrained(path, dtype=dtype, device=device)


def _pidenex_load(path, dtype, device):
    from tah_b200.models.pidenex import PidenexForCausalLM
    return PidenexForCausalLM.from_pretrained(path, dtype=dtype, device=device)


def _is(class_name: str) -> Callable[[object], bool]:
    return lambda model: type(model).__name__ == class_name


def _hybrid_engine(model, **kw):
    from tah_b200.engine.hybrid import HybridEngine
    return HybridEngine(model, **kw)


register_family(Family("qwen3-tah", _qwen3_matches, _qwen3_load, _qwen3_owns, _qwen3_engine))
register_family(Family("gunuvik", lambda c: c.get("architecture") == "Gunuvik", _gunuvik_load, _is("GunuvikForCausalLM"),
                       _hybrid_engine, "gunuvik"))
register_family(Family("ditilix", lambda c: c.get("architecture") == "Ditilix", _ditilix_load, _is("DitilixForCausalLM"),
                       _hybrid_engine, "ditilix"))
register_family(Family("niralix", lambda c: c.get("architecture") == "Niralix", _niralix_load, _is("NiralixForCausalLM"),
                       _hybrid_engine, "niralix"))
register_family(Family("pidenex", lambda c: c.get("architecture") == "Pidenex", _pidenex_load, _is("PidenexForCausalLM"),
                       _hybrid_engine, "pidenex"))
