"""Checkpoint directories of layer-stack models: model.safetensors, or shards named by model.safetensors.index.json,
checked against the family's tensor catalog (every name, every shape, nothing beyond) before anything is read."""
from __future__ import annotations

import json
import os
from typing import Dict, Tuple

import torch

from .safetensors_io import SafetensorsError, SafetensorsFile


class StackCheckpoint:
    def __init__(self, directory: str, shapes: Dict[str, Tuple[int, ...]]):
        index = os.path.join(directory, "model.safetensors.index.json")
        if os.path.exists(index):
            with open(index) as f:
                names = sorted(set(json.load(f)["weight_map"].values()))
        else:
            names = ["model.safetensors"]
        self.where: Dict[str, SafetensorsFile] = {}
        for n in names:
            f = SafetensorsFile(os.path.join(directory, n))
            for t in f.names():
                if t in self.where:
                    raise SafetensorsError(f"{directory}: tensor '{t}' appears twice")
                self.where[t] = f
        missing, unknown = sorted(set(shapes) - set(self.where)), sorted(set(self.where) - set(shapes))
        if missing or unknown:
            raise SafetensorsError(f"{directory}: missing tensors {missing[:4]}, unknown tensors {unknown[:4]} "
                                   f"({len(missing)} / {len(unknown)} in all)")
        for t, shape in shapes.items():
            e = self.where[t].entries[t]
            if tuple(e.shape) != tuple(shape):
                raise SafetensorsError(f"{directory}: tensor '{t}' has shape {list(e.shape)}, expected {list(shape)}")
            if e.dtype not in ("BF16", "F16", "F32"):
                raise SafetensorsError(f"{directory}: tensor '{t}' has dtype {e.dtype}")

    def read(self, name: str) -> torch.Tensor:
        return self.where[name].read(name)
