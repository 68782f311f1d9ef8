"""One table from an architecture's name to its configuration and model spec.

The reference selects the architecture with a ``match`` on the name string
and a tuple of per-architecture defaults (src/model/config.rs:136-150,
241-351).  Here an architecture is one row: a function that parses
``config.json`` into its typed configuration and a function that lays that
configuration out as a :class:`~.spec.ModelSpec`.
"""

from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Any, Callable, Dict, Mapping, Tuple

from .spec import ConfigError, ModelSpec


@dataclass(frozen=True)
class Architecture:
    name: str
    parse_config: Callable[[Mapping[str, Any]], Any]
    build_spec: Callable[[Any], ModelSpec]
    # (config.json, {tensor name: shape}) -> config.json completed with the sizes that only a
    # model folder's tensors give; None: config.json says everything
    sizes_from_tensors: Any = None


_ARCHITECTURES: Dict[str, Architecture] = {}


def register_architecture(names, parse_config, build_spec, sizes_from_tensors=None) -> None:
    """Add a row.  ``names`` are the strings config.json may carry in
    ``architectures`` or ``model_type``."""
    if isinstance(names, str):
        names = (names,)
    arch = Architecture(names[0], parse_config, build_spec, sizes_from_tensors)
    for n in names:
        _ARCHITECTURES[n] = arch


def known_architectures() -> Tuple[str, ...]:
    return tuple(sorted(_ARCHITECTURES))


def architecture_of(config: Mapping[str, Any]) -> Architecture:
    """Find the row for a config.json dictionary."""
    names = list(config.get("architectures") or [])
    for key in ("architecture", "model_type"):
        if config.get(key):
            names.append(config[key])
    if not names:
        raise ConfigError("config.json: none of 'architectures', 'architecture' and 'model_type' is given; "
                          f"known architectures: {', '.join(known_architectures())}")
    for n in names:
        if n in _ARCHITECTURES:
            return _ARCHITECTURES[n]
    raise ConfigError(f"unsupported architecture {', '.join(map(repr, names))}; "
                      f"known architectures: {', '.join(known_architectures())}")


def read_config_json(model_dir: str) -> dict:
    path = os.path.join(model_dir, "config.json")
    if not os.path.isfile(path):
        raise ConfigError(f"{path}: no such file")
    with open(path) as f:
        try:
            return json.load(f)
        except json.JSONDecodeError as e:
            raise ConfigError(f"{path}: not valid JSON ({e})") from None


def spec_from_config(config: Mapping[str, Any],
                     shapes: Mapping[str, Tuple[int, ...]] = None) -> Tuple[Any, ModelSpec]:
    """config.json dictionary -> (typed configuration, model spec).  ``shapes``: the shapes of
    a model folder's tensors by name, for architectures some of whose sizes only they give."""
    arch = architecture_of(config)
    if shapes is not None and arch.sizes_from_tensors is not None:
        config = arch.sizes_from_tensors(config, shapes)
    typed = arch.parse_config(config)
    return typed, arch.build_spec(typed)


def _register_builtin() -> None:
    from .gemma2 import Gemma2Config, gemma2_spec
    register_architecture(("Gemma2ForCausalLM", "gemma2"), Gemma2Config.from_dict, gemma2_spec)
    from .karupel import KarupelConfig, karupel_spec
    register_architecture(("Karupel", "karupel"), KarupelConfig.from_dict, karupel_spec)
    from .vavupel import VavupelConfig, vavupel_spec
    register_architecture(("Vavupel", "vavupel"), VavupelConfig.from_dict, vavupel_spec)
    from .gegorax import GegoraxConfig, gegorax_sizes, gegorax_spec
    register_architecture(("Gegorax", "gegorax"), GegoraxConfig.from_dict, gegorax_spec, gegorax_sizes)
    from .besorax import BesoraxConfig, besorax_sizes, besorax_spec
    register_architecture(("Besorax", "besorax"), BesoraxConfig.from_dict, besorax_spec, besorax_sizes)
    from .kerolorn import KerolornConfig, kerolorn_sizes, kerolorn_spec
    register_architecture(("Kerolorn", "kerolorn"), KerolornConfig.from_dict, kerolorn_spec, kerolorn_sizes)
    from .simetar import SimetarConfig, simetar_sizes, simetar_spec
    register_architecture(("Simetar", "simetar"), SimetarConfig.from_dict, simetar_spec, simetar_sizes)


_register_builtin()
