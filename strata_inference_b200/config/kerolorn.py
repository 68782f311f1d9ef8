"""Kerolorn: the typed configuration and its translation into a ModelSpec.

A Kerolorn model is a list of layers that config.json writes out one by one:

    {"architecture": "Kerolorn", "vocab": V, "width": W, "norm": {"eps": e},
     "canon": {"taps": n}, "logit_scale": s,
     "layers": [{"type": "attention", "mixer": {...}, "mlp": {...} | null}]}

``mixer`` = {heads, kv_heads, dim, vdim, scale, rot: {dims, base, scaling: {factor, original,
fast, slow}}, mask: {size, keep_first}}; ``mlp`` = {"kind": "moe", "router": {experts, top,
scale}, "expert": {ff}, "shared": {ff}}.  ``rot``, ``rot.scaling``, ``mask``, ``keep_first`` and
``shared`` may be absent.

What the design fixes and config.json has no key for is stated once in :func:`kerolorn_spec`:
RMS norms before and after each sub-layer, x <- x + norm1b(mixer(norm1(x))), then x <- x +
norm2b(ff(norm2(x))); between norm1 and the mixer a short causal convolution per channel is
added to its own input; grouped-query softmax attention without biases, neighbouring pairs
rotated, q and k divided by their root mean square per head AFTER the rotation, a stored factor
per head on the scores, a window of the last ``size`` positions that also keeps the sequence's
first ``keep_first``; routed experts of gate, up and down matrices with SiLU, chosen by the
softmax over all experts plus a stored correction, weighed by that softmax without the
correction times ``router.scale``; a shared expert of the same form weighed by the sigmoid of
one number per row.  The logits have a matrix of their own and are multiplied by
``logit_scale``.  Tensor names: ``embed``, ``l<i>.norm1`` / ``norm1b`` / ``norm2`` / ``norm2b``,
``l<i>.canon1``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List, Mapping, Optional, Tuple

from .spec import ConfigError, LayerSpec, ModelSpec, PartSpec, ScheduleEntry, require

_TYPES = ("attention",)
# positions a sequence may reach where config.json sets no bound ("max_positions")
_DEFAULT_POSITIONS = 1 << 20


def _positive(d: Any, key: str, where: str) -> int:
    v = d.get(key) if isinstance(d, Mapping) else None
    if isinstance(v, bool) or not isinstance(v, int) or v <= 0:
        raise ConfigError(f"config.json: {where}.'{key}' must be a positive integer, got {v!r}")
    return v


def _number(d: Any, key: str, where: str, positive: bool = False) -> float:
    v = d.get(key) if isinstance(d, Mapping) else None
    if isinstance(v, bool) or not isinstance(v, (int, float)) or (positive and v <= 0):
        raise ConfigError(f"config.json: {where}.'{key}' must be a {'positive ' if positive else ''}number, "
                          f"got {v!r}")
    return float(v)


def _mapping(d: Any, key: str, where: str) -> Mapping[str, Any]:
    v = d.get(key) if isinstance(d, Mapping) else None
    if not isinstance(v, Mapping):
        raise ConfigError(f"config.json: {where}.'{key}' is missing")
    return v


def _rot(m: Mapping[str, Any], where: str, width: int) -> Optional[Dict[str, Any]]:
    """The rotation of a mixer: {"dims", "base", "scaling" (None or four numbers)}, or None when
    nothing is rotated."""
    rot = m.get("rot")
    if not rot:
        return None
    where += ".rot"
    dims, base = _positive(rot, "dims", where), _number(rot, "base", where, positive=True)
    if dims % 2 or dims > width:
        raise ConfigError(f"config.json: {where}: 'dims' = {dims} must be even and at most the "
                          f"head's width ({width})")
    scaling = None
    if rot.get("scaling"):
        scaling = {k: _number(rot["scaling"], k, where + ".scaling", positive=True)
                   for k in ("factor", "original", "fast", "slow")}
        if base == 1.0:
            raise ConfigError(f"config.json: {where}: a scaled rotation needs a 'base' other than 1")
    return {"dims": dims, "base": base, "scaling": scaling}


def _attention(m: Mapping[str, Any], where: str) -> Dict[str, Any]:
    out: Dict[str, Any] = {"heads": _positive(m, "heads", where), "dim": _positive(m, "dim", where),
                           "vdim": _positive(m, "vdim", where), "scale": _number(m, "scale", where)}
    out["kv_heads"] = _positive(m, "kv_heads", where) if m.get("kv_heads") is not None else out["heads"]
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(f"config.json: {where}: {out['heads']} heads cannot share "
                          f"{out['kv_heads']} kv_heads")
    out["rot"] = _rot(m, where, out["dim"])
    out["window"] = out["keep_first"] = 0
    mask = m.get("mask")
    if mask:
        out["window"] = _positive(mask, "size", where + ".mask")
        keep = mask.get("keep_first") or 0
        if isinstance(keep, bool) or not isinstance(keep, int) or keep < 0:
            raise ConfigError(f"config.json: {where}.mask.'keep_first' must be an integer of at least 0, "
                              f"got {keep!r}")
        out["keep_first"] = keep
    return out


def _mlp(mlp: Any, where: str) -> Optional[Dict[str, Any]]:
    if not mlp:
        return None
    kind = mlp.get("kind", "moe") if isinstance(mlp, Mapping) else None
    if kind != "moe":
        raise ConfigError(f"config.json: {where}.'kind' = {kind!r} is not 'moe'")
    router, expert = _mapping(mlp, "router", where), _mapping(mlp, "expert", where)
    out = {"experts": _positive(router, "experts", where + ".router"),
           "top": _positive(router, "top", where + ".router"),
           "scale": _number(router, "scale", where + ".router") if router.get("scale") is not None else 1.0,
           "ff": _positive(expert, "ff", where + ".expert"), "shared": 0}
    if out["top"] > out["experts"]:
        raise ConfigError(f"config.json: {where}.router: 'top' exceeds 'experts'")
    if mlp.get("shared"):
        out["shared"] = _positive(mlp["shared"], "ff", where + ".shared")
    return out


@dataclass(frozen=True)
class KerolornLayer:
    type: str
    mixer: Mapping[str, Any]                 # checked sizes and constants of the mixer
    mlp: Optional[Mapping[str, Any]]         # None: no feed-forward


@dataclass(frozen=True)
class KerolornConfig:
    vocab: int
    width: int
    eps: float
    taps: int
    logit_scale: float
    layers: Tuple[KerolornLayer, ...]
    max_positions: int
    raw: Mapping[str, Any]

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "KerolornConfig":
        vocab, width = require(d, "vocab", int), require(d, "width", int)
        if vocab <= 0 or width <= 0:
            raise ConfigError("config.json: 'vocab' and 'width' must be positive")
        eps = _number(require(d, "norm"), "eps", "norm", positive=True)
        taps = _positive(require(d, "canon"), "taps", "canon")
        logit_scale = float(require(d, "logit_scale", float))
        listed = require(d, "layers")
        if not isinstance(listed, (list, tuple)) or not listed:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers: List[KerolornLayer] = []
        for i, l in enumerate(listed):
            where = f"layers[{i}]"
            kind = l.get("type") if isinstance(l, Mapping) else None
            if kind not in _TYPES:
                raise ConfigError(f"config.json: {where}.'type' = {kind!r} is not one of "
                                  f"{', '.join(_TYPES)}")
            layers.append(KerolornLayer(kind, _attention(_mapping(l, "mixer", where), where + ".mixer"),
                                        _mlp(l.get("mlp"), where + ".mlp")))
        most = d.get("max_positions")
        return cls(vocab=vocab, width=width, eps=eps, taps=taps, logit_scale=logit_scale, layers=tuple(layers),
                   max_positions=_DEFAULT_POSITIONS if most is None else _positive(d, "max_positions", ""),
                   raw=dict(d))

    def to_dict(self) -> dict:
        return dict(self.raw)


def kerolorn_sizes(config: Mapping[str, Any], shapes: Mapping[str, Tuple[int, ...]]) -> dict:
    """config.json completed with the sizes that it leaves to a folder's tensors: a size that
    config.json gives stays as it is; one that it omits is read off the shape of the tensor that
    has it."""
    out = copy.deepcopy(dict(config))

    def rows(name):
        shape = shapes.get(name)
        return int(shape[0]) if shape else 0

    def cols(name):
        shape = shapes.get(name)
        return int(shape[1]) if shape and len(shape) == 2 else 0

    def fill(d, key, value):
        if isinstance(d, dict) and d.get(key) is None and value:
            d[key] = int(value)
    fill(out, "vocab", rows("embed"))
    fill(out, "width", cols("embed"))
    if out.get("canon") is None and cols("l0.canon1"):
        out["canon"] = {}
    fill(out.get("canon"), "taps", cols("l0.canon1"))
    for i, l in enumerate(out.get("layers") or []):
        if not isinstance(l, dict):
            continue
        m, pre = l.get("mixer"), f"l{i}.mix."
        if isinstance(m, dict):
            fill(m, "heads", rows(pre + "temp"))
            H = m.get("heads")
            if isinstance(H, int) and not isinstance(H, bool) and H > 0:
                fill(m, "dim", rows(pre + "q") // H)
                fill(m, "vdim", cols(pre + "o") // H)
                if isinstance(m.get("dim"), int) and m["dim"] > 0:
                    fill(m, "kv_heads", rows(pre + "k") // m["dim"])
        mlp, pre = l.get("mlp"), f"l{i}.mlp."
        if isinstance(mlp, dict):
            mlp.setdefault("router", {})
            mlp.setdefault("expert", {})
            fill(mlp["router"], "experts", rows(pre + "router"))
            fill(mlp["expert"], "ff", rows(pre + "e0.gate"))
            if mlp.get("shared") is None and rows(pre + "shared.gate"):
                mlp["shared"] = {}
            if isinstance(mlp.get("shared"), dict):
                fill(mlp["shared"], "ff", rows(pre + "shared.gate"))
    return out


_ATTENTION_NAMES = {"q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "temp": "temp",
                    "o_proj.weight": "o"}
_NORM_SITES = {"pre_mixer": "norm1", "post_mixer": "norm1b", "pre_feed_forward": "norm2",
               "post_feed_forward": "norm2b"}


def _moe_names(n_experts: int) -> Dict[str, str]:
    names = {"router.weight": "router", "correction": "correction", "shared.gate.weight": "shared.sg"}
    for part in ("gate", "up", "down"):
        names[f"shared.{part}_proj.weight"] = f"shared.{part}"
        for e in range(n_experts):
            names[f"experts.{e}.{part}_proj.weight"] = f"e{e}.{part}"
    return names


def kerolorn_spec(cfg: KerolornConfig) -> ModelSpec:
    """Lay the configuration out as parts, layer by layer."""
    norm = PartSpec("rms_norm", {"eps": cfg.eps})
    layers, schedule, tolerated = [], [], []
    for i, l in enumerate(cfg.layers):
        m = l.mixer
        rot = m["rot"]
        position = PartSpec("rope_interleaved", {"theta": rot["base"], "rotary_dim": rot["dims"],
                                                 "frequencies": "float64", "yarn": rot["scaling"]}) \
            if rot else PartSpec("none", {})
        mixer = PartSpec("attention", {
            "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
            "value_dim": m["vdim"], "score_scale": m["scale"], "logit_softcap": 0.0,
            "window": m["window"], "keep_first": m["keep_first"] if m["window"] else 0,
            "qk_norm": {"eps": cfg.eps, "weight": False, "after_rotation": True},
            "head_temp": True, "position": position})
        ffn: Optional[PartSpec] = None
        ff_names: Mapping[str, str] = {}
        norms = {"pre_mixer": norm, "post_mixer": norm}
        if l.mlp:
            ffn = PartSpec("routed_experts", {
                "experts": l.mlp["experts"], "top": l.mlp["top"], "intermediate_size": l.mlp["ff"],
                "form": "gated_silu", "score": "softmax_all", "router_bias": False, "correction": True,
                "router_scale": l.mlp["scale"],
                "shared": {"intermediate_size": l.mlp["shared"], "gate": True} if l.mlp["shared"] else None})
            ff_names = _moe_names(l.mlp["experts"])
            norms.update({"pre_feed_forward": norm, "post_feed_forward": norm})
        else:
            # a folder may still hold the norms of the sub-layer that is not there
            tolerated += [f"l{i}.norm2", f"l{i}.norm2b"]
        sites = {"mixer": "mix.", "feed_forward": "mlp.", "mixer_input": "canon1"}
        sites.update(_NORM_SITES)
        tensor_names: Dict[str, Mapping[str, str]] = {"mixer": _ATTENTION_NAMES, "feed_forward": ff_names,
                                                      "mixer_input": {"weight": ""}}
        tensor_names.update({site: {"weight": ""} for site in _NORM_SITES})
        layers.append(LayerSpec(prefix=f"l{i}.", block="sandwich", mixer=mixer, feed_forward=ffn,
                                norms=norms, names=sites, tensor_names=tensor_names,
                                mixer_input=PartSpec("short_conv", {"taps": cfg.taps})))
        schedule.append(ScheduleEntry(i))
    spec = ModelSpec(
        architecture="Kerolorn", hidden_size=cfg.width, vocab_size=cfg.vocab,
        max_positions=cfg.max_positions,
        embedding=PartSpec("token_embedding", {"scale": 1.0}),
        layers=tuple(layers), schedule=tuple(schedule), final_norm=norm,
        head=PartSpec("lm_head", {"tied": False, "logit_softcap": 0.0, "logit_scale": cfg.logit_scale}),
        names={"embedding": "", "final_norm": "final.norm", "head": "head"},
        tensor_names={"embedding": {"weight": "embed"}, "final_norm": {"weight": ""}, "head": {"weight": ""}},
        tolerated=tuple(tolerated), stop_tokens=())
    spec.validate()
    return spec
