"""Model families: how the engine and the tools find the classes that serve a configuration.

A family is chosen by the type of its configuration (``family_of``) or by what a checkpoint says about itself
(``open_model``: a folder whose config.json names an ``architecture``, or a W8A8 safetensors file)."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable

from . import layered_config as LC
from .config import PRESETS as W8A8_PRESETS
from .config import ModelConfig, RuntimeConfig


@dataclass(frozen=True)
class Family:
    name: str
    config: type
    dtypes: tuple[str, ...]
    model: Callable                # (cfg, rt, weights, comm, device, tp_ctx=) -> decoder
    random_weights: Callable       # (cfg, rt, rank, device, seed) -> weights
    load: Callable                 # (path, rt, rank, device) -> (cfg, weights)


def _w8a8() -> Family:
    from . import weights as Wt
    from .decoder import Decoder
    return Family("w8a8", ModelConfig, ("bfloat16",), Decoder,
                  lambda cfg, rt, rank, device, seed: Wt.random_shard(cfg, rt.tp, rank, device, seed),
                  lambda path, rt, rank, device: Wt.load_shard(path, rt.tp, rank, device))


def _layered() -> Family:
    from . import layered_weights as LW
    from .layered import LayeredDecoder
    return Family("layered", LC.LayeredConfig, ("bfloat16", "float32"), LayeredDecoder,
                  lambda cfg, rt, rank, device, seed: LW.random_weights(cfg, rt, device, seed),
                  lambda path, rt, rank, device: LW.load(path, rt, device))


ARCHITECTURES = {name: _layered for name in LC.DESIGNS}       # config.json "architecture" -> family
PRESETS = {**W8A8_PRESETS, "volonex-8b": LC.volonex_8b, "volonex-1b": LC.volonex_1b, "tiny-volonex": LC.tiny_volonex,
           "rakelorn-16b": LC.rakelorn_16b, "rakelorn-2b": LC.rakelorn_2b, "tiny-rakelorn": LC.tiny_rakelorn}


def family_of(cfg) -> Family:
    for make in (_w8a8, _layered):
        f = make()
        if isinstance(cfg, f.config):
            return f
    raise TypeError(f"no model family for a {type(cfg).__name__}")


def family_at(path: str) -> Family:
    """The family of a checkpoint on disk."""
    if os.path.isdir(path):
        with open(os.path.join(path, "config.json")) as f:
            arch = json.load(f).get("architecture")
        if arch not in ARCHITECTURES:
            raise ValueError(f"unknown architecture {arch!r} (known: {', '.join(ARCHITECTURES)})")
        return ARCHITECTURES[arch]()
    return _w8a8()


def open_model(path: str, rt: RuntimeConfig, device, rank: int = 0):
    """Checkpoint on disk -> (cfg, weights)."""
    f = family_at(path)
    if rt.dtype not in f.dtypes:
        raise ValueError(f"the {f.name} models have no {rt.dtype} form")
    return f.load(path, rt, rank, device)
