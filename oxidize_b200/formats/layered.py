"""Checkpoint directories that list their layers one by one: ``config.json`` with ``"architecture"`` and a ``"layers"``
list, and ``*.safetensors`` beside it (one file or several shards).

The class shows the part of :class:`~oxidize_b200.formats.gguf.GGUFFile`'s surface that model loading, ``show`` /
``inspect`` and the autotuner's fingerprint use, so that such a directory is accepted wherever a GGUF path is."""
from __future__ import annotations

import glob
import json
import os
from dataclasses import dataclass
from typing import Any, Dict, Tuple, Union

import numpy as np

from .gguf import GGUFFile, load_gguf
from .safetensors_io import SafeTensorsFile, load_sharded


@dataclass(frozen=True)
class _TypeName:
    name: str


@dataclass(frozen=True)
class LayeredTensorInfo:
    name: str
    shape: Tuple[int, ...]
    type: _TypeName
    nbytes: int


class LayeredCheckpoint:
    version = 1
    alignment = 8

    def __init__(self, path: str):
        self.path = os.path.normpath(path)
        with open(os.path.join(path, "config.json"), encoding="utf-8") as f:
            self.config: Dict[str, Any] = json.load(f)
        self.architecture = str(self.config["architecture"]).lower()
        files = sorted(glob.glob(os.path.join(path, "*.safetensors")))
        if not files:
            raise FileNotFoundError(f"{path} has a config.json but no .safetensors files")
        self._where: Dict[str, Tuple[SafeTensorsFile, str]] = load_sharded(files)
        self.tensors: Dict[str, LayeredTensorInfo] = {}
        for name, (f, key) in self._where.items():
            dt, shape, b, e = f.entries[key]
            self.tensors[name] = LayeredTensorInfo(name, shape, _TypeName(dt), e - b)
        self.metadata: Dict[str, Any] = {"general.architecture": self.architecture, "general.name": os.path.basename(self.path)}
        self.metadata.update({k: v for k, v in self.config.items() if isinstance(v, (int, float, str, bool))})

    def get(self, key: str, default=None):
        return self.metadata.get(key, default)

    def has_tensor(self, name: str) -> bool:
        return name in self.tensors

    def advise(self, willneed: bool = False, hugepages: bool = False) -> None:
        """(The file mapping of this format takes no access hints.)"""

    def raw(self, name: str) -> Tuple[np.ndarray, str]:
        """(typed view, dtype name); BF16 comes as uint16 bit patterns."""
        if name not in self._where:
            raise KeyError(f"{self.path}: tensor {name!r} is missing")
        f, key = self._where[name]
        return f.tensor(key), f.dtype(key)


def is_layered_checkpoint(path: str) -> bool:
    cfg = os.path.join(path, "config.json")
    if not os.path.isfile(cfg):
        return False
    try:
        with open(cfg, encoding="utf-8") as f:
            c = json.load(f)
    except ValueError:
        return False
    return isinstance(c, dict) and isinstance(c.get("architecture"), str) and isinstance(c.get("layers"), list)


Checkpoint = Union[GGUFFile, LayeredCheckpoint]


def open_checkpoint(path: str) -> Checkpoint:
    return LayeredCheckpoint(path) if os.path.isdir(path) and is_layered_checkpoint(path) else load_gguf(path)
