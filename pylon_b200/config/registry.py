"""One registry from an architecture's name (``config.json`` ``architectures[0]``) to its
typed configuration class and the function that describes its model.

raun6k/Pylon serves one hard-gated checkpoint (src/pylon/model/config.py:7,35-49) and has
no registry; here the name chooses, and an unknown name is an error that lists the known.
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Any, Callable, Mapping, Optional

from pylon_b200.config.model_config import ConfigError, FikeraxConfig, PinedraConfig, Qwen3Config, RirusunConfig, VopepelConfig, ZabusunConfig, ZemavikConfig
from pylon_b200.parts.spec import ModelSpec


@dataclass(frozen=True)
class Architecture:
    name: str
    config_class: Any                                   # has from_dict(mapping) and to_dict()
    build_spec: Callable[[Any, Optional[int]], ModelSpec]  # (config, max_positions) -> ModelSpec


ARCHITECTURES: dict[str, Architecture] = {}


def register_architecture(name: str, config_class: Any, build_spec: Callable[[Any, Optional[int]], ModelSpec]) -> None:
    ARCHITECTURES[name] = Architecture(name, config_class, build_spec)


def architecture_of(data: Mapping[str, Any]) -> Architecture:
    names = data.get("architectures")
    if names is None and isinstance(data.get("architecture"), str):   # some formats name their one architecture in the singular
        names = [data["architecture"]]
    if not isinstance(names, (list, tuple)) or len(names) != 1 or not isinstance(names[0], str):
        raise ConfigError(f"config.json 'architectures' (or 'architecture') must name exactly one architecture, got {names!r}")
    if names[0] not in ARCHITECTURES:
        raise ConfigError(f"unknown architecture '{names[0]}' (known: {', '.join(sorted(ARCHITECTURES))})")
    return ARCHITECTURES[names[0]]


def read_config(model_dir: str | Path) -> tuple[Architecture, Any]:
    """Reads ``model_dir/config.json``; returns the architecture entry and its typed config."""
    path = Path(model_dir) / "config.json"
    if not path.is_file():
        raise ConfigError(f"{path} does not exist")
    try:
        data = json.loads(path.read_text())
    except json.JSONDecodeError as error:
        raise ConfigError(f"{path} is not valid JSON: {error}") from error
    if not isinstance(data, dict):
        raise ConfigError(f"{path} must hold a JSON object")
    architecture = architecture_of(data)
    return architecture, architecture.config_class.from_dict(data)


def _register_builtin() -> None:
    from pylon_b200.models.qwen3 import qwen3_spec

    register_architecture(Qwen3Config.architecture, Qwen3Config, qwen3_spec)
    from pylon_b200.models.vopepel import vopepel_spec

    register_architecture(VopepelConfig.architecture, VopepelConfig, vopepel_spec)
    from pylon_b200.models.fikerax import fikerax_spec

    register_architecture(FikeraxConfig.architecture, FikeraxConfig, fikerax_spec)
    from pylon_b200.models.zemavik import zemavik_spec

    register_architecture(ZemavikConfig.architecture, ZemavikConfig, zemavik_spec)
    from pylon_b200.models.rirusun import rirusun_spec

    register_architecture(RirusunConfig.architecture, RirusunConfig, rirusun_spec)
    from pylon_b200.models.zabusun import zabusun_spec

    register_architecture(ZabusunConfig.architecture, ZabusunConfig, zabusun_spec)
    from pylon_b200.models.pinedra import pinedra_spec

    register_architecture(PinedraConfig.architecture, PinedraConfig, pinedra_spec)


_register_builtin()
