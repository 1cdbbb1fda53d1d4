"""Architectures the framework knows by name, and how a checkpoint folder turns into one of them.

An entry names the configuration class (``from_dict`` reads the fields of a ``config.json``) and, for
architectures the serving engine runs, where their serving model lives (imported on first use, so that
reading a configuration needs no kernels).
"""
from __future__ import annotations

import importlib
import json
import os
from dataclasses import dataclass
from typing import Dict, Optional


@dataclass(frozen=True)
class Architecture:
    name: str
    config: str                    # "module:class"
    serving: Optional[str] = None  # "module:class"
    parts: Optional[str] = None    # part of the native libraries its serving model needs (see rumus_b200/build.py)

    def _load(self, ref: str):
        mod, cls = ref.split(":")
        return getattr(importlib.import_module(mod), cls)

    def config_class(self):
        return self._load(self.config)

    def serving_class(self):
        if self.serving is None:
            raise ValueError(f"architecture {self.name!r} has no serving model")
        return self._load(self.serving)


_ARCHS: Dict[str, Architecture] = {}


def register(name: str, config: str, serving: Optional[str] = None, parts: Optional[str] = None) -> None:
    _ARCHS[name] = Architecture(name, config, serving, parts)


def architecture(name: str) -> Architecture:
    if name not in _ARCHS:
        raise ValueError(f"unknown architecture {name!r}; known: {', '.join(sorted(_ARCHS))}")
    return _ARCHS[name]


def architecture_of(config) -> Architecture:
    """The entry whose configuration class ``config`` is an instance of."""
    for a in _ARCHS.values():
        if type(config).__name__ == a.config.split(":")[1]:
            return a
    raise ValueError(f"{type(config).__name__} belongs to no registered architecture")


def read_config_json(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def load_config(folder: str):
    """Configuration object of a checkpoint folder (``config.json`` names its ``architecture``)."""
    d = read_config_json(folder)
    if "architecture" not in d:
        raise ValueError(f"{folder}/config.json names no architecture")
    return architecture(d["architecture"]).config_class().from_dict(d)


register("GPT", "rumus_b200.models.gpt:GPTConfig")
register("Llama", "rumus_b200.models.llama:LlamaConfig", "rumus_b200.serve.llama:Int4LlamaShard")
register("Zidalix", "rumus_b200.models.zidalix:ZidalixConfig", "rumus_b200.serve.zidalix:ZidalixServing", parts="latent")
register("Nufupel", "rumus_b200.models.nufupel:NufupelConfig", "rumus_b200.serve.nufupel:NufupelServing", parts="window")
register("Potodra", "rumus_b200.models.potodra:PotodraConfig", "rumus_b200.serve.potodra:PotodraServing", parts="hybrid")
register("Lerosun", "rumus_b200.models.lerosun:LerosunConfig", "rumus_b200.serve.lerosun:LerosunServing", parts="talk")
