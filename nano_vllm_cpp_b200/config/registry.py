"""One registry from an architecture's name (``architectures[0]`` of config.json, or its ``architecture``
string) to its configuration class and its model builder.

The reference has no such table: its runner owns one model class by value
(include/nanovllm/model_runner.hpp:29) and never reads ``architectures``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Callable

from .model_config import ConfigError, read_config_json


@dataclass(frozen=True)
class Architecture:
    name: str
    config_from_dict: Callable[[dict], Any]       # dict of config.json -> typed config
    build_model: Callable[..., Any]               # (config) -> parts.model.ModelSpec


_ARCHITECTURES: dict[str, Architecture] = {}


def register_architecture(name: str, config_from_dict, build_model) -> None:
    _ARCHITECTURES[name] = Architecture(name, config_from_dict, build_model)


def known_architectures() -> list[str]:
    _ensure_builtin()
    return sorted(_ARCHITECTURES)


def get_architecture(name: str) -> Architecture:
    _ensure_builtin()
    try:
        return _ARCHITECTURES[name]
    except KeyError:
        raise ConfigError(f"unknown architecture {name!r}; known: {', '.join(sorted(_ARCHITECTURES))}") from None


def load_model_config(model_dir: str):
    """Read ``config.json`` and return ``(architecture, typed config)``."""
    d = read_config_json(model_dir)
    arch = get_architecture(architecture_name(d))
    return arch, arch.config_from_dict(d)


def architecture_name(d: dict) -> str:
    """The model class a config.json names: the first of ``architectures``, or the string ``architecture``."""
    archs = d.get("architectures")
    if isinstance(archs, list) and archs and isinstance(archs[0], str):
        return archs[0]
    if isinstance(d.get("architecture"), str):
        return d["architecture"]
    raise ConfigError("config.json: key 'architectures' must be a non-empty list of names "
                      "(or 'architecture' a name)")


def _ensure_builtin() -> None:
    # The built-in architectures register themselves on import.
    from ..models import qwen2_moe, bizodra, kifunex, sanesun, gekitar, sevelorn, dubarax  # noqa: F401
