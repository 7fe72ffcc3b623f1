"""Which model class, weight layout and loader a configuration belongs to.  The engine, the trace replay, the command line and
the benchmarks all choose through here."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, Optional, Tuple

from .config import (BobaraxConfig, LugizenConfig, ModelConfig, NubosunConfig, TinapelConfig, from_hf_config, parse_bobarax_config, parse_lugizen_config,
                     parse_nubosun_config, parse_tinapel_config)


@dataclass(frozen=True)
class Architecture:
    name: str
    config_type: type
    model: Callable[[], type]              # imported on use: the model modules need the native library
    dtypes: Tuple[str, ...]                # compute types the model runs in
    tensor_parallel: bool
    parse: Optional[Callable[[dict], object]] = None   # config.json that names this architecture (None: the HF layout)


def _llama():
    from .llama import LlamaTP
    return LlamaTP


def _nubosun():
    from .nubosun import Nubosun
    return Nubosun


def _tinapel():
    from .tinapel import Tinapel
    return Tinapel


def _bobarax():
    from .bobarax import Bobarax
    return Bobarax


def _lugizen():
    from .lugizen import Lugizen
    return Lugizen


ARCHITECTURES = {
    "llama": Architecture("llama", ModelConfig, _llama, ("bfloat16",), True),
    "nubosun": Architecture("nubosun", NubosunConfig, _nubosun, ("bfloat16", "float32"), False, parse_nubosun_config),
    "tinapel": Architecture("tinapel", TinapelConfig, _tinapel, ("bfloat16", "float32"), False, parse_tinapel_config),
    "bobarax": Architecture("bobarax", BobaraxConfig, _bobarax, ("bfloat16", "float32"), False, parse_bobarax_config),
    "lugizen": Architecture("lugizen", LugizenConfig, _lugizen, ("bfloat16", "float32"), False, parse_lugizen_config),
}


def architecture_of(cfg) -> Architecture:
    for a in ARCHITECTURES.values():
        if isinstance(cfg, a.config_type):
            return a
    raise ValueError(f"no architecture for a configuration of type {type(cfg).__name__}")


def load_config(model_dir: str):
    """Configuration object of a model directory, its kind chosen by ``config.json``."""
    path = os.path.join(model_dir, "config.json")
    with open(path) as f:
        c = json.load(f)
    arch = str(c.get("architecture", "")).lower()
    if arch in ARCHITECTURES and ARCHITECTURES[arch].parse is not None:
        return ARCHITECTURES[arch].parse(c)
    if arch:
        raise ValueError(f"unknown architecture {c['architecture']!r}")
    return from_hf_config(path)            # Llama / Qwen2 families in the HF layout
