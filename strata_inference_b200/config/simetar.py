"""Simetar: the typed configuration and its translation into a ModelSpec.

A Simetar model is a list of layers that config.json writes out one by one:

    {"architecture": "Simetar", "vocab": V, "width": W, "norm": {"eps": e},
     "layers": [{"type": "attention" | "latent_attention", "mixer": {...}, "mlp": {...} | null}]}

attention: {heads, kv_heads, dim, vdim, conv, scale, softcap, mask: {size}, rot: {dims, base,
scaling: {factor, low, high, original}}}; latent_attention: {heads, dim, rot_dim, vdim, kv_rank, scale,
kv_from, rot: {dims, base, scaling: {factor, original, fast, slow}}}; ``mlp`` = {"kind": "dense", "ff"}.
``rot``, ``rot.scaling``, ``mask``, ``softcap`` and ``kv_from`` may be absent.

What the design fixes and config.json has no key for is stated once in :func:`simetar_spec`: a
sub-layer reads the residual stream itself and passes a layer norm (weight and bias) on its way
out, x <- x + norm1(mixer(x)), x <- x + norm2(ff(x)).  The attention layers' q and k have biases,
pass a short causal convolution over time per channel, are normed as whole rows and rotated in
neighbouring pairs; the values are the keys as the convolution leaves them; one is added to
the softmax's denominator.  The latent attention layers rotate in half-split pairs, with YaRN;
one with ``kv_from`` has no down projection and reads the rows that the named layer caches.
Both multiply the concatenated heads by a gate per element ahead of the output product.  The
feed-forward is gated with the tanh form of gelu; the logits have a matrix of their own.
Tensor names: ``embed``, ``l<i>.norm1`` / ``norm2`` (biases: ``.b`` behind), ``l<i>.mix.*``,
``l<i>.mlp.*``, ``final.norm``, ``head``.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List, Mapping, Optional, Tuple

from .spec import ConfigError, LayerSpec, ModelSpec, PartSpec, ScheduleEntry, require

_TYPES = ("attention", "latent_attention")
# positions a sequence may reach where config.json sets no bound ("max_positions")
_DEFAULT_POSITIONS = 1 << 20
# the score of every attention layer's sink: e^0 = 1 joins the softmax's denominator
SINK_SCORE = 0.0


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


def _rot(m: Mapping[str, Any], where: str, width: int, scaling_keys: Tuple[str, ...]) -> Optional[Dict[str, Any]]:
    """The rotation of a mixer: {"dims", "base", "scaling" (None or its numbers)}, or None when
    nothing is rotated."""
    rot = m.get("rot")
    if not rot:
        return None
    where += ".rot"
    dims, base = _positive(rot, "dims", where), _number(rot, "base", where, positive=True)
    if dims % 2 or dims > width:
        raise ConfigError(f"config.json: {where}: 'dims' = {dims} must be even and at most the "
                          f"rotated width ({width})")
    scaling = None
    if rot.get("scaling"):
        scaling = {k: _number(rot["scaling"], k, where + ".scaling", positive=True) for k in scaling_keys}
        if base == 1.0 and "fast" in scaling:
            raise ConfigError(f"config.json: {where}: a scaled rotation needs a 'base' other than 1")
    return {"dims": dims, "base": base, "scaling": scaling}


def _attention(m: Mapping[str, Any], where: str) -> Dict[str, Any]:
    out: Dict[str, Any] = {"heads": _positive(m, "heads", where), "dim": _positive(m, "dim", where),
                           "conv": _positive(m, "conv", where), "scale": _number(m, "scale", where)}
    out["kv_heads"] = _positive(m, "kv_heads", where) if m.get("kv_heads") is not None else out["heads"]
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(f"config.json: {where}: {out['heads']} heads cannot share "
                          f"{out['kv_heads']} kv_heads")
    if m.get("vdim") is not None and _positive(m, "vdim", where) != out["dim"]:
        raise ConfigError(f"config.json: {where}: values are keys, so 'vdim' = {m['vdim']} must be 'dim' = {out['dim']}")
    out["rot"] = _rot(m, where, out["dim"], ("factor", "low", "high", "original"))
    out["window"] = _positive(m["mask"], "size", where + ".mask") if m.get("mask") else 0
    out["softcap"] = _number(m, "softcap", where, positive=True) if m.get("softcap") else 0.0
    return out


def _latent(m: Mapping[str, Any], where: str) -> Dict[str, Any]:
    out: Dict[str, Any] = {k: _positive(m, k, where) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank")}
    out["scale"] = _number(m, "scale", where)
    out["rot"] = _rot(m, where, out["rot_dim"], ("factor", "original", "fast", "slow"))
    src = m.get("kv_from")
    if src is not None and (isinstance(src, bool) or not isinstance(src, int) or src < 0):
        raise ConfigError(f"config.json: {where}.'kv_from' must name a layer, got {src!r}")
    out["kv_from"] = src
    return out


def _mlp(mlp: Any, where: str) -> Optional[Dict[str, Any]]:
    if not mlp:
        return None
    kind = mlp.get("kind", "dense") if isinstance(mlp, Mapping) else None
    if kind != "dense":
        raise ConfigError(f"config.json: {where}.'kind' = {kind!r} is not 'dense'")
    return {"ff": _positive(mlp, "ff", where)}


@dataclass(frozen=True)
class SimetarLayer:
    type: str
    mixer: Mapping[str, Any]                 # checked sizes and constants of the mixer
    mlp: Optional[Mapping[str, Any]]         # None: no feed-forward


@dataclass(frozen=True)
class SimetarConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[SimetarLayer, ...]
    max_positions: int
    raw: Mapping[str, Any]

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "SimetarConfig":
        vocab, width = require(d, "vocab", int), require(d, "width", int)
        if vocab <= 0 or width <= 0:
            raise ConfigError("config.json: 'vocab' and 'width' must be positive")
        eps = _number(require(d, "norm"), "eps", "norm", positive=True)
        listed = require(d, "layers")
        if not isinstance(listed, (list, tuple)) or not listed:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers: List[SimetarLayer] = []
        for i, l in enumerate(listed):
            where = f"layers[{i}]"
            kind = l.get("type") if isinstance(l, Mapping) else None
            if kind not in _TYPES:
                raise ConfigError(f"config.json: {where}.'type' = {kind!r} is not one of "
                                  f"{', '.join(_TYPES)}")
            mixer = (_attention if kind == "attention" else _latent)(_mapping(l, "mixer", where), where + ".mixer")
            layers.append(SimetarLayer(kind, mixer, _mlp(l.get("mlp"), where + ".mlp")))
        for i, l in enumerate(layers):
            src = l.mixer.get("kv_from")
            if src is None:
                continue
            where = f"layers[{i}].mixer.'kv_from' = {src}"
            if src >= i or layers[src].type != "latent_attention" or layers[src].mixer["kv_from"] is not None:
                raise ConfigError(f"config.json: {where} must name an earlier latent attention layer with a "
                                  f"down projection of its own")
            for key in ("kv_rank", "rot_dim", "rot"):
                if layers[src].mixer[key] != l.mixer[key]:
                    raise ConfigError(f"config.json: {where}: '{key}' differs between the two layers")
        most = d.get("max_positions")
        return cls(vocab=vocab, width=width, eps=eps, layers=tuple(layers),
                   max_positions=_DEFAULT_POSITIONS if most is None else _positive(d, "max_positions", ""),
                   raw=dict(d))

    def to_dict(self) -> dict:
        return dict(self.raw)


def simetar_sizes(config: Mapping[str, Any], shapes: Mapping[str, Tuple[int, ...]]) -> dict:
    """config.json completed with the sizes that it leaves to a folder's tensors: a size that
    config.json gives stays as it is; one that it omits is read off the shape of the tensor that
    has it (head counts cannot be, and stay required)."""
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
    layers = out.get("layers") or []
    for i, l in enumerate(layers):
        if not isinstance(l, dict):
            continue
        m, pre = l.get("mixer"), f"l{i}.mix."
        H = m.get("heads") if isinstance(m, dict) else None
        if isinstance(H, int) and not isinstance(H, bool) and H > 0:
            if l.get("type") == "attention":
                fill(m, "dim", rows(pre + "q") // H)
                fill(m, "conv", cols(pre + "q.conv"))
                if isinstance(m.get("dim"), int) and m["dim"] > 0:
                    fill(m, "kv_heads", rows(pre + "k") // m["dim"])
            elif l.get("type") == "latent_attention":
                fill(m, "kv_rank", cols(pre + "uk"))
                fill(m, "dim", rows(pre + "uk") // H)
                fill(m, "vdim", rows(pre + "uv") // H)
                if isinstance(m.get("dim"), int):
                    fill(m, "rot_dim", rows(pre + "q") // H - m["dim"])
        if isinstance(l.get("mlp"), dict):
            fill(l["mlp"], "ff", rows(f"l{i}.mlp.gate"))
    return out


_NORM_NAMES = {"weight": "", "b": ".b"}
_ATTENTION_NAMES = {"q_proj.weight": "q", "k_proj.weight": "k", "q_proj.bias": "q.b", "k_proj.bias": "k.b",
                    "q_conv.weight": "q.conv", "k_conv.weight": "k.conv", "q_norm.weight": "q.norm",
                    "k_norm.weight": "k.norm", "gate_proj.weight": "g", "o_proj.weight": "o"}
_LATENT_NAMES = {"q_proj.weight": "q", "dkv_proj.weight": "dkv", "dkv_norm.weight": "dkv.norm",
                 "uk_proj.weight": "uk", "uv_proj.weight": "uv", "gate_proj.weight": "g", "o_proj.weight": "o"}
_DENSE_NAMES = {"gate_proj.weight": "gate", "up_proj.weight": "up", "down_proj.weight": "down"}
_NORM_SITES = {"post_mixer": "norm1", "post_feed_forward": "norm2"}


def simetar_spec(cfg: SimetarConfig) -> ModelSpec:
    """Lay the configuration out as parts, layer by layer; a layer that reads another's rows
    becomes a schedule entry that names the lender's."""
    norm, plain = PartSpec("layer_norm", {"eps": cfg.eps}), PartSpec("identity", {})
    lenders = {l.mixer.get("kv_from") for l in cfg.layers}
    layers, schedule, tolerated = [], [], []
    for i, l in enumerate(cfg.layers):
        m, rot = l.mixer, l.mixer["rot"]
        lender = None
        if l.type == "attention":
            position = PartSpec("rope_interleaved", {
                "theta": rot["base"], "rotary_dim": rot["dims"], "frequencies": "float64",
                "llama3": rot["scaling"]}) if rot else PartSpec("none", {})
            mixer = PartSpec("attention", {
                "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
                "value_dim": m["dim"], "values_from_keys": True, "bias": True, "qk_conv": m["conv"],
                "qk_norm": {"eps": cfg.eps, "whole": True}, "position": position, "score_scale": m["scale"],
                "logit_softcap": m["softcap"], "exact_cap": True, "window": m["window"],
                "sink_score": SINK_SCORE, "output_gate": True})
            names = _ATTENTION_NAMES
        else:
            lender = m["kv_from"]
            position = PartSpec("rope_neox", {
                "theta": rot["base"], "rotary_dim": rot["dims"], "frequencies": "float64",
                "yarn": rot["scaling"]}) if rot else PartSpec("none", {})
            mixer = PartSpec("latent_attention", {
                "num_heads": m["heads"], "head_dim": m["dim"], "rot_dim": m["rot_dim"],
                "value_dim": m["vdim"], "kv_rank": m["kv_rank"], "score_scale": m["scale"], "window": 0,
                "norm_eps": cfg.eps, "position": position, "output_gate": True,
                "borrows_cache": lender is not None, "lends_cache": i in lenders})
            names = _LATENT_NAMES
        ffn: Optional[PartSpec] = None
        ff_names: Mapping[str, str] = {}
        norms = {"pre_mixer": plain, "post_mixer": norm}
        if l.mlp:
            ffn = PartSpec("gated_mlp", {"intermediate_size": l.mlp["ff"], "activation": "gelu_pytorch_tanh"})
            ff_names = _DENSE_NAMES
            norms.update({"pre_feed_forward": plain, "post_feed_forward": norm})
        else:
            # a folder may still hold the norm of the sub-layer that is not there
            tolerated += [f"l{i}.norm2", f"l{i}.norm2.b"]
        sites = {"mixer": "mix.", "feed_forward": "mlp.", "pre_mixer": "", "pre_feed_forward": ""}
        sites.update(_NORM_SITES)
        tensor_names: Dict[str, Mapping[str, str]] = {"mixer": names, "feed_forward": ff_names}
        tensor_names.update({site: _NORM_NAMES for site in _NORM_SITES})
        layers.append(LayerSpec(prefix=f"l{i}.", block="sandwich", mixer=mixer, feed_forward=ffn,
                                norms=norms, names=sites, tensor_names=tensor_names))
        schedule.append(ScheduleEntry(i, cache_of=lender))
    spec = ModelSpec(
        architecture="Simetar", hidden_size=cfg.width, vocab_size=cfg.vocab,
        max_positions=cfg.max_positions,
        embedding=PartSpec("token_embedding", {"scale": 1.0}),
        layers=tuple(layers), schedule=tuple(schedule), final_norm=norm,
        head=PartSpec("lm_head", {"tied": False, "logit_softcap": 0.0}),
        names={"embedding": "", "final_norm": "final.norm", "head": "head"},
        tensor_names={"embedding": {"weight": "embed"}, "final_norm": _NORM_NAMES, "head": {"weight": ""}},
        tolerated=tuple(tolerated), stop_tokens=())
    spec.validate()
    return spec
