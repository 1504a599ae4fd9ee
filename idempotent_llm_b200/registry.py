"""The one registry from an architecture's name (config.json ``architectures[0]``)
to its typed configuration and its model.

The reference has a single hard-wired class and a backend alias table that
raises on unknown names (src/detllm/backends.py:17-34); the same
normalise-or-raise behaviour is kept here for architecture names.

An entry holds the configuration class (``from_dict``, ``to_dict``,
``to_model_spec``) and a builder ``(model_spec, weights, runtime) -> model``.
The default builder assembles the generic decoder from registered parts.
"""

from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, Dict, Optional

from .config.specs import ConfigError


@dataclass(frozen=True)
class Architecture:
    name: str
    config_class: type
    build_model: Optional[Callable] = None  # None: the generic assembly from parts


_ARCHITECTURES: Dict[str, Architecture] = {}


def register_architecture(name: str, config_class: type, build_model: Optional[Callable] = None) -> None:
    for attr in ("from_dict", "to_model_spec"):
        if not hasattr(config_class, attr):
            raise TypeError(f"configuration class for {name!r} lacks {attr}()")
    _ARCHITECTURES[name] = Architecture(name, config_class, build_model)


def architecture(name: str) -> Architecture:
    try:
        return _ARCHITECTURES[name]
    except KeyError:
        raise ConfigError(f"unknown architecture {name!r}; registered: {sorted(_ARCHITECTURES)}") from None


def registered_architectures():
    return sorted(_ARCHITECTURES)


def read_config(model_dir: str):
    """Read ``model_dir/config.json`` and return (Architecture, typed configuration)."""
    path = os.path.join(model_dir, "config.json")
    if not os.path.isfile(path):
        raise ConfigError(f"{path} does not exist")
    with open(path) as f:
        raw = json.load(f)
    arch = architecture(architecture_name(raw, path))
    return arch, arch.config_class.from_dict(raw)


def architecture_name(raw: dict, where: str = "config.json") -> str:
    """The name a config.json gives its architecture: the first of ``architectures`` (a list), or
    ``architecture`` (one name)."""
    archs = raw.get("architectures")
    if archs:
        return archs[0]
    if isinstance(raw.get("architecture"), str) and raw["architecture"]:
        return raw["architecture"]
    raise ConfigError(f"{where}: key 'architectures' (or 'architecture') is missing or empty")


def _register_builtin() -> None:
    from .config.qwen3 import ARCHITECTURE, Qwen3Config
    register_architecture(ARCHITECTURE, Qwen3Config)
    from .config.lunulix import ARCHITECTURE as LUNULIX, LunulixConfig
    register_architecture(LUNULIX, LunulixConfig)
    from .config.panodra import ARCHITECTURE as PANODRA, PanodraConfig
    register_architecture(PANODRA, PanodraConfig)
    from .config.fuginex import ARCHITECTURE as FUGINEX, FuginexConfig
    register_architecture(FUGINEX, FuginexConfig)
    from .config.pununex import ARCHITECTURE as PUNUNEX, PununexConfig
    register_architecture(PUNUNEX, PununexConfig)
    from .config.tosodra import ARCHITECTURE as TOSODRA, TosodraConfig
    register_architecture(TOSODRA, TosodraConfig)
    from .config.zazulix import ARCHITECTURE as ZAZULIX, ZazulixConfig
    register_architecture(ZAZULIX, ZazulixConfig)


_register_builtin()
