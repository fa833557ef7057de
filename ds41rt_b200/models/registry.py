"""Model families by configuration: which configuration class, weight loader and engine a model directory or a preset name
stands for.  The command line, the server and `bin/trace_run` all choose their model class here."""
from __future__ import annotations

import json
import os
from typing import Dict, List, Optional

from ..config import ModelConfig
from . import belasun, genesun


class UnsupportedDtype(ValueError):
    """The family has no engine for the requested number format."""


class Family:
    name = ""
    presets: tuple = ()
    dtypes: tuple = ("bf16",)

    def matches(self, doc: dict) -> bool:
        raise NotImplementedError

    def config(self, doc: dict, text: str, name: str):
        raise NotImplementedError

    def preset(self, name: str, layers: int = 0):
        raise NotImplementedError

    def engine(self, cfg, weights, **kw):
        raise NotImplementedError


class DS41Family(Family):
    """DeepSeek-V4.1-Flash-shaped models (models/ds41.py)."""
    name = "ds41"
    presets = ("tiny", "small", "flash")

    def matches(self, doc):
        return "text_config" in doc

    def config(self, doc, text, name):
        return ModelConfig.from_official_json(text)

    def preset(self, name, layers=0):
        if name == "flash":
            return ModelConfig.flash(layers or 4)
        return ModelConfig.small() if name == "small" else ModelConfig.tiny()

    def load_weights(self, directory, cfg, device, dtype="bf16", rank=0, world=1, expert_dtype="mxfp8"):
        if dtype != "bf16":
            raise UnsupportedDtype(f"{self.name}: no {dtype} engine")
        from ..loader.official import load_engine_weights
        return load_engine_weights(directory, cfg, rank, world, device, expert_dtype=expert_dtype)

    def random_weights(self, cfg, device, seed=0, dtype="bf16", rank=0, world=1, expert_dtype="mxfp8"):
        if dtype != "bf16":
            raise UnsupportedDtype(f"{self.name}: no {dtype} engine")
        from .ds41 import EngineWeights
        return EngineWeights.random(cfg, rank, world, device, seed=seed, expert_dtype=expert_dtype)

    def engine(self, cfg, weights, fabric=None, **kw):
        from .ds41 import DS41Engine
        return DS41Engine(cfg, weights, fabric, **kw)


class StackFamily(Family):
    """Layer-stack models (models/stack.py); `module` reads the family's configuration and names its tensors."""
    dtypes = ("bf16", "f32")

    def __init__(self, name: str, module):
        self.name, self.module, self.presets = name, module, module.PRESETS

    def matches(self, doc):
        return self.module.matches(doc)

    def config(self, doc, text, name):
        return self.module.parse(doc, name)

    def preset(self, name, layers=0):
        return self.module.preset(name, layers or None)

    def tensor_shapes(self, cfg):
        return self.module.tensor_shapes(cfg)

    def layer_shapes(self, cfg, layer: int):
        return self.module.layer_shapes(cfg, layer)

    def _one_rank(self, world):
        if world != 1:
            raise ValueError("layer-stack models run on one GPU")

    def load_weights(self, directory, cfg, device, dtype="bf16", rank=0, world=1, expert_dtype=None):
        from ..loader.stack import StackCheckpoint
        self._one_rank(world)
        return self.module.build_weights(cfg, StackCheckpoint(directory, self.tensor_shapes(cfg)).read, device, dtype)

    def random_weights(self, cfg, device, seed=0, dtype="bf16", rank=0, world=1, expert_dtype=None):
        self._one_rank(world)
        return self.module.random_weights(cfg, device, seed, dtype)

    def engine(self, cfg, weights, fabric=None, kv_dtype="bf16", **kw):
        from .stack import StackEngine
        if kv_dtype != "bf16":
            raise ValueError("layer-stack models keep bf16 (or 32-bit) cache rows")
        return StackEngine(cfg, weights, **kw)


FAMILIES: Dict[str, Family] = {f.name: f for f in (DS41Family(), StackFamily("genesun", genesun),
                                                  StackFamily("belasun", belasun))}
PRESETS: List[str] = [p for f in FAMILIES.values() for p in f.presets]


def family_of(cfg) -> Family:
    return FAMILIES["ds41"] if isinstance(cfg, ModelConfig) else FAMILIES[cfg.family]


def config_from_file(path: str):
    """config.json (a file, or the directory that holds it) -> (family, configuration)."""
    if os.path.isdir(path):
        path = os.path.join(path, "config.json")
    with open(path) as f:
        text = f.read()
    doc = json.loads(text)
    for fam in FAMILIES.values():
        if fam.matches(doc):
            return fam, fam.config(doc, text, os.path.basename(os.path.dirname(os.path.abspath(path))) or fam.name)
    raise ValueError(f"{path}: no model family reads this configuration")


def preset(name: str, layers: int = 0):
    for fam in FAMILIES.values():
        if name in fam.presets:
            return fam, fam.preset(name, layers)
    raise ValueError(f"unknown model {name!r}")


def load_engine(directory: str, device, dtype: str = "bf16", **engine_args):
    """Engine of the model in `directory` (config.json and its safetensors files)."""
    fam, cfg = config_from_file(directory)
    if dtype not in fam.dtypes:
        raise UnsupportedDtype(f"{fam.name}: no {dtype} engine")
    return fam.engine(cfg, fam.load_weights(directory, cfg, device, dtype), **engine_args)
