"""Architecture-neutral description of a decoder: what the engine builds from.

An architecture's typed configuration (read from its own ``config.json``
keys) is translated into a :class:`ModelSpec`.  From there on nothing knows
the architecture's name: the engine looks up each :class:`PartSpec`'s
``kind`` in the part registries (``parts/registry.py``) and hands it its
``params``.

The reference expresses the same choices as per-architecture default tuples
and per-layer flags inside one config struct (src/model/config.rs:59-123,
241-351, 379-385); here they are data, layer by layer.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Mapping, Optional, Tuple


class ConfigError(ValueError):
    """A configuration that cannot be built; the message names the key."""


@dataclass(frozen=True)
class PartSpec:
    """One part of a layer: the registered ``kind`` and its sizes and constants."""

    kind: str
    params: Mapping[str, Any] = field(default_factory=dict)

    def __getitem__(self, key: str) -> Any:
        return self.params[key]

    def get(self, key: str, default: Any = None) -> Any:
        return self.params.get(key, default)


@dataclass(frozen=True)
class LayerSpec:
    """One decoder layer: which block arrangement and which parts fill it.

    ``prefix`` is the common start of the layer's tensor names and ``names``
    gives, for each site of the block ("mixer", "feed_forward" and the norm
    sites), what follows it; a part only knows its own local names (such as
    ``q_proj.weight``) and never sees the whole name table.
    ``norms`` maps the block arrangement's norm sites to norm specs.
    ``feed_forward`` None: the layer is its mixer alone.
    ``tensor_names`` (optional) gives, per site, stored names for the part's local names
    where a model folder calls them otherwise ({"mixer": {"q_proj.weight": "q"}} stores the
    mixer's ``q_proj.weight`` as ``<prefix><names["mixer"]>q``).
    """

    prefix: str
    block: str
    mixer: PartSpec
    feed_forward: Optional[PartSpec]
    norms: Mapping[str, PartSpec]
    names: Mapping[str, str]
    tensor_names: Mapping[str, Mapping[str, str]] = field(default_factory=dict)
    # a registered "tail": a part that runs behind the sub-layers on the stream itself
    # (``names["tail"]`` is what follows the layer's prefix in its tensors' names)
    tail: Optional[PartSpec] = None
    # a registered "mixer_input": a part that works on the mixer's (normed) input rows and may keep
    # state of its own per schedule entry (``names["mixer_input"]`` is what follows the prefix)
    mixer_input: Optional[PartSpec] = None
    # parameters of the block arrangement itself (``residual_scale`` of the pre-norm block)
    block_params: Mapping[str, Any] = field(default_factory=dict)


@dataclass(frozen=True)
class ScheduleEntry:
    """One run of a layer.  ``layer`` indexes :attr:`ModelSpec.layers` (the
    same index may appear more than once: the weights are then shared).
    ``cache_of`` names an earlier schedule entry whose keys and values (or
    state) this run reads instead of writing its own.  ``begins_pass``: before this
    run the residual stream is mixed with the embedding's output by the model's
    ``pass_mix`` part (a model whose layers are walked several times does this at
    the start of every pass)."""

    layer: int
    cache_of: Optional[int] = None
    begins_pass: bool = False


@dataclass(frozen=True)
class ModelSpec:
    architecture: str
    hidden_size: int
    vocab_size: int
    max_positions: int
    embedding: PartSpec
    layers: Tuple[LayerSpec, ...]
    schedule: Tuple[ScheduleEntry, ...]
    final_norm: PartSpec
    head: PartSpec
    names: Mapping[str, str] = field(default_factory=dict)  # "embedding", "final_norm", "head"
    stop_tokens: Tuple[int, ...] = ()
    # stored names for local names, per site, as in LayerSpec.tensor_names
    tensor_names: Mapping[str, Mapping[str, str]] = field(default_factory=dict)
    # the part that runs before every schedule entry with ``begins_pass`` (a registered
    # "joint": forward(h, x0) -> h), named by ``names["pass_mix"]``
    pass_mix: Optional[PartSpec] = None
    # stored tensors that a model folder may hold although nothing reads them
    tolerated: Tuple[str, ...] = ()

    def validate(self) -> None:
        if self.hidden_size <= 0 or self.vocab_size <= 0 or self.max_positions <= 0:
            raise ConfigError("hidden_size, vocab_size and max_positions must be positive")
        if not self.layers:
            raise ConfigError("a model needs at least one layer")
        for pos, e in enumerate(self.schedule):
            if not 0 <= e.layer < len(self.layers):
                raise ConfigError(f"schedule[{pos}] names layer {e.layer}, "
                                  f"but there are {len(self.layers)} layers")
            if e.begins_pass and self.pass_mix is None:
                raise ConfigError(f"schedule[{pos}] begins a pass, but the model has no 'pass_mix' part")
            if e.cache_of is not None:
                if not 0 <= e.cache_of < pos:
                    raise ConfigError(f"schedule[{pos}].cache_of={e.cache_of} must name "
                                      f"an earlier schedule entry")
                if self.schedule[e.cache_of].cache_of is not None:
                    raise ConfigError(f"schedule[{pos}].cache_of={e.cache_of} names an entry "
                                      f"that itself borrows a cache")


def require(d: Mapping[str, Any], key: str, typ=None) -> Any:
    """Fetch a required config.json key; the error names it."""
    if key not in d or d[key] is None:
        raise ConfigError(f"config.json: required key '{key}' is missing")
    v = d[key]
    if typ is int and (isinstance(v, bool) or not isinstance(v, int)):
        raise ConfigError(f"config.json: key '{key}' must be an integer, got {v!r}")
    if typ is float and (isinstance(v, bool) or not isinstance(v, (int, float))):
        raise ConfigError(f"config.json: key '{key}' must be a number, got {v!r}")
    return v
