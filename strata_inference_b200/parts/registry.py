"""Registries of parts by ``kind``.

``register_mixer("my_kind", MyMixer)`` makes ``PartSpec("my_kind", {...})``
buildable anywhere a mixer is expected; the same holds for feed-forwards,
norms, position encodings, blocks, embeddings and heads.  The built-in
parts register themselves when ``strata_inference_b200.parts`` is imported.
"""

from __future__ import annotations

from typing import Callable, Dict

from ..config.spec import ConfigError, PartSpec

_REGISTRIES: Dict[str, Dict[str, type]] = {
    "mixer": {}, "feed_forward": {}, "norm": {}, "position": {},
    "block": {}, "embedding": {}, "head": {}, "joint": {}, "tail": {},
    "mixer_input": {},
}


def _register(role: str, kind: str, cls: type) -> type:
    _REGISTRIES[role][kind] = cls
    return cls


def register_mixer(kind: str, cls: type) -> type:
    return _register("mixer", kind, cls)


def register_feed_forward(kind: str, cls: type) -> type:
    return _register("feed_forward", kind, cls)


def register_norm(kind: str, cls: type) -> type:
    return _register("norm", kind, cls)


def register_position(kind: str, cls: type) -> type:
    return _register("position", kind, cls)


def register_block(kind: str, cls: type) -> type:
    return _register("block", kind, cls)


def register_embedding(kind: str, cls: type) -> type:
    return _register("embedding", kind, cls)


def register_head(kind: str, cls: type) -> type:
    return _register("head", kind, cls)


def register_joint(kind: str, cls: type) -> type:
    """A part that joins two streams into one: ``forward(h, x0) -> h``."""
    return _register("joint", kind, cls)


def register_tail(kind: str, cls: type) -> type:
    """A part that runs behind a layer's sub-layers, on the stream itself: ``forward(x, ctx) -> y``
    with ``gain`` and ``eps`` of the RMS norm that y passes before it is added."""
    return _register("tail", kind, cls)


def register_mixer_input(kind: str, cls: type) -> type:
    """A part between a layer's first norm and its mixer: ``forward(x, ctx, entry) -> x'``, with
    ``state_need()`` for what it keeps per slot and schedule entry."""
    return _register("mixer_input", kind, cls)


def part_class(role: str, kind: str) -> type:
    table = _REGISTRIES[role]
    if kind not in table:
        raise ConfigError(f"no {role} of kind '{kind}' is registered; "
                          f"known: {', '.join(sorted(table)) or '(none)'}")
    return table[kind]


def known(role: str):
    return tuple(sorted(_REGISTRIES[role]))
