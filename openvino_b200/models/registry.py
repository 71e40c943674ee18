"""Checkpoint folders (``config.json`` + ``model.safetensors``): the architecture that ``config.json`` names selects the reader of
its configuration and the names of its tensors; everything else (weights in kernel layout, cache, scheduling, sampling) is the
serving program's. Graph models (IR, ONNX, ...) do not pass through here: see frontend/ and runtime/llm_import.py.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, Dict

from ..utils.safetensors import SafetensorsFile
from . import busatar, sapasun
from .llm_config import LayeredConfig


@dataclass(frozen=True)
class Architecture:
    read_config: Callable[[dict], LayeredConfig]
    tensor_name: Callable[[int, str, str], str]
    tensor_shapes: Callable[[LayeredConfig], dict]


ARCHITECTURES: Dict[str, Architecture] = {"Busatar": Architecture(busatar.read_config, busatar.tensor_name, busatar.tensor_shapes),
                                          "Sapasun": Architecture(sapasun.read_config, sapasun.tensor_name, sapasun.tensor_shapes)}


def register(name: str, arch: Architecture) -> None:
    ARCHITECTURES[name] = arch


@dataclass
class Checkpoint:
    """A configuration and where its tensors come from."""
    config: LayeredConfig
    arch: Architecture
    tensors: object            # mapping name -> torch.Tensor

    def __post_init__(self):
        self._shapes = self.arch.tensor_shapes(self.config)

    def __call__(self, layer: int, part: str, key: str):
        name = self.arch.tensor_name(layer, part, key)
        try:
            t = self.tensors[name]
        except KeyError:
            raise KeyError("the checkpoint has no tensor '%s'" % name) from None
        want = tuple(self._shapes[name])      # None: a size that the configuration leaves to the tensor
        if len(t.shape) != len(want) or any(w is not None and n != w for n, w in zip(t.shape, want)):
            raise ValueError("tensor '%s' has the shape %s, its configuration asks for %s" % (name, tuple(t.shape), want))
        return t


def is_checkpoint_dir(path: str) -> bool:
    return os.path.isfile(os.path.join(path, "config.json")) and os.path.isfile(os.path.join(path, "model.safetensors"))


def load_checkpoint(path: str) -> Checkpoint:
    with open(os.path.join(path, "config.json")) as f:
        cfg = json.load(f)
    return from_dict(cfg, SafetensorsFile(os.path.join(path, "model.safetensors")))


def from_dict(cfg: dict, tensors) -> Checkpoint:
    """The same from a parsed configuration and any name -> tensor mapping."""
    name = cfg.get("architecture")
    if name not in ARCHITECTURES:
        raise ValueError("unknown architecture '%s' (known: %s)" % (name, ", ".join(sorted(ARCHITECTURES))))
    arch = ARCHITECTURES[name]
    return Checkpoint(arch.read_config(cfg), arch, tensors)
