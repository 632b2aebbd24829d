"""Architectures the engine serves: where a model's configuration and weights come from, and which class runs it.

A model is named by a GGUF file (``deepseek2``), by a folder with ``config.json`` and safetensors files (the configuration's
``architecture`` key selects the entry), by hyper-parameters, or by the name of a random-weight preset.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Any, Callable, Dict, Optional

from . import lugovik, nibalix, rupatar, zomavik
from .deepseek2 import DeepSeek2Model
from .hparams import ARCH as DEEPSEEK2, DeepSeek2HParams
from .hparams import preset as _deepseek2_preset


@dataclass(frozen=True)
class Architecture:
    name: str
    hparams: type
    model: type
    preset: Callable[[str], Any]
    # folder checkpoints: hyper-parameters of a folder, (name, tensor) pairs of a folder; None: the architecture comes as GGUF
    load_config: Optional[Callable[[str], Any]] = None
    iter_checkpoint: Optional[Callable[[str, Any], Any]] = None
    iter_random: Optional[Callable[..., Any]] = None
    sharded: bool = False             # tensor / expert parallelism over several GPUs


ARCHITECTURES: Dict[str, Architecture] = {
    DEEPSEEK2: Architecture(DEEPSEEK2, DeepSeek2HParams, DeepSeek2Model, _deepseek2_preset, sharded=True),
    nibalix.ARCH: Architecture(nibalix.ARCH, nibalix.NibalixHParams, nibalix.NibalixModel, nibalix.preset, nibalix.load_config,
                               nibalix.iter_checkpoint, nibalix.iter_random),
    lugovik.ARCH: Architecture(lugovik.ARCH, lugovik.LugovikHParams, lugovik.LugovikModel, lugovik.preset, lugovik.load_config,
                               lugovik.iter_checkpoint, lugovik.iter_random),
    zomavik.ARCH: Architecture(zomavik.ARCH, zomavik.ZomavikHParams, zomavik.ZomavikModel, zomavik.preset, zomavik.load_config,
                               zomavik.iter_checkpoint, zomavik.iter_random),
    rupatar.ARCH: Architecture(rupatar.ARCH, rupatar.RupatarHParams, rupatar.RupatarModel, rupatar.preset, rupatar.load_config,
                               rupatar.iter_checkpoint, rupatar.iter_random),
}


def is_folder_model(path: Optional[str]) -> bool:
    return bool(path) and os.path.isfile(os.path.join(path, "config.json"))


def for_path(path: str) -> Architecture:
    """The architecture of a model file or folder."""
    if not is_folder_model(path):
        return ARCHITECTURES[DEEPSEEK2]
    with open(os.path.join(path, "config.json")) as f:
        name = json.load(f).get("architecture")
    a = ARCHITECTURES.get(name)
    if a is None or a.load_config is None:
        raise ValueError(f"{path}: architecture {name!r} is not served from a folder "
                         f"(known: {', '.join(k for k, v in ARCHITECTURES.items() if v.load_config)}; convert others to GGUF)")
    return a


def for_hparams(hp: Any) -> Architecture:
    for a in ARCHITECTURES.values():
        if isinstance(hp, a.hparams):
            return a
    raise TypeError(f"no architecture for {type(hp).__name__}")


def preset(name: str):
    """Hyper-parameters of a named random-weight preset of any architecture."""
    for a in ARCHITECTURES.values():
        try:
            return a.preset(name)
        except KeyError:
            continue
    raise KeyError(name)
