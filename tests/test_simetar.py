"""Simetar on the CPU: the configuration and its layout as parts, and the plain model's own mechanisms
(tests/plain_simetar.py) against closed forms."""

from __future__ import annotations

import copy
import math

import numpy as np
import pytest
import torch

import plain_simetar as plain
from simetar_cases import (ALONE, MIXED, ODD, SHARP, WIDE, attention, dense, latent, llama3, model, random_model,
                           random_weights, yarn)

from strata_inference_b200.config.registry import spec_from_config
from strata_inference_b200.config.spec import ConfigError
from strata_inference_b200.engine.model import expected_tensors, resident_plan


def test_every_size_and_constant_comes_from_the_configuration():
    typed, spec = spec_from_config(MIXED)
    assert spec.architecture == "Simetar" and spec.hidden_size == 64 and spec.vocab_size == 200
    assert not spec.head["tied"] and spec.embedding["scale"] == 1.0
    first, second, third, reader = spec.layers[:4]
    assert first.block == "sandwich"
    assert {s: n.kind for s, n in first.norms.items()} == {
        "pre_mixer": "identity", "post_mixer": "layer_norm", "pre_feed_forward": "identity", "post_feed_forward": "layer_norm"}
    assert first.norms["post_mixer"]["eps"] == 1e-5 and spec.final_norm.kind == "layer_norm"
    m = first.mixer
    assert (m["num_heads"], m["num_kv_heads"], m["head_dim"], m["value_dim"]) == (4, 2, 16, 16)
    assert (m["window"], m["score_scale"], m["logit_softcap"], m["qk_conv"]) == (37, 0.2, 15.0, 3)
    assert m["values_from_keys"] and m["bias"] and m["output_gate"] and m["exact_cap"] and m["sink_score"] == 0.0
    assert m["qk_norm"] == {"eps": 1e-5, "whole": True}
    assert m["position"].kind == "rope_interleaved" and m["position"]["rotary_dim"] == 8
    assert m["position"]["llama3"] == llama3() and third.mixer["position"]["llama3"] is None
    assert spec.layers[5].mixer["window"] == 0 and spec.layers[5].mixer["logit_softcap"] == 0.0
    m = second.mixer
    assert (m["num_heads"], m["head_dim"], m["rot_dim"], m["value_dim"], m["kv_rank"]) == (4, 16, 8, 24, 40)
    assert m["position"].kind == "rope_neox" and m["position"]["yarn"] == yarn() and m["output_gate"]
    assert m["lends_cache"] and not m["borrows_cache"] and spec.layers[4].mixer["lends_cache"]
    assert reader.mixer["borrows_cache"] and not reader.mixer["lends_cache"] and reader.mixer["score_scale"] == 0.2
    assert [e.cache_of for e in spec.schedule] == [None, None, None, 1, None, None, 1, 4]
    assert third.feed_forward is None and "post_feed_forward" not in third.norms
    assert first.feed_forward.kind == "gated_mlp" and first.feed_forward["intermediate_size"] == 96
    assert first.feed_forward["activation"] == "gelu_pytorch_tanh"


@pytest.mark.parametrize("cfg", [MIXED, ODD, WIDE, SHARP] + [ALONE[k] for k in sorted(ALONE)] + [random_model(s) for s in range(8)])
def test_tensor_table_matches_the_random_weights(cfg):
    _, spec = spec_from_config(cfg)
    table = expected_tensors(spec)
    w = random_weights(cfg, seed=1)
    needed = {n for n, d in table.items() if not d.optional}
    assert needed == set(w), (sorted(needed - set(w)), sorted(set(w) - needed))
    for n in needed:
        assert tuple(table[n].shape) == tuple(w[n].shape), n
    placed = {prefix + q.source for res, prefix in resident_plan(spec).values() for q in res.pieces}
    assert placed == needed


def _edit(path, value):
    def edit(c):
        d = c
        for k in path[:-1]:
            d = d[k]
        if value is None:
            d.pop(path[-1])
        else:
            d[path[-1]] = value
    return edit


@pytest.mark.parametrize("edit, text", [
    (_edit(["norm"], None), "norm"),
    (_edit(["norm", "eps"], 0), "norm.'eps'"),
    (_edit(["layers", 0, "type"], "recurrent"), "layers[0].'type'"),
    (_edit(["layers", 0, "mixer", "scale"], "x"), "layers[0].mixer.'scale'"),
    (_edit(["layers", 0, "mixer", "conv"], 0), "layers[0].mixer.'conv'"),
    (_edit(["layers", 0, "mixer", "kv_heads"], 3), "kv_heads"),
    (_edit(["layers", 0, "mixer", "vdim"], 24), "'vdim'"),
    (_edit(["layers", 0, "mixer", "softcap"], -1.0), "layers[0].mixer.'softcap'"),
    (_edit(["layers", 0, "mixer", "rot", "dims"], 7), "layers[0].mixer.rot"),
    (_edit(["layers", 0, "mixer", "rot", "scaling", "high"], None), "layers[0].mixer.rot.scaling.'high'"),
    (_edit(["layers", 1, "mixer", "rot", "scaling", "slow"], None), "layers[1].mixer.rot.scaling.'slow'"),
    (_edit(["layers", 1, "mixer", "rot", "dims"], 10), "layers[1].mixer.rot"),
    (_edit(["layers", 0, "mixer", "mask", "size"], 0), "layers[0].mixer.mask.'size'"),
    (_edit(["layers", 0, "mlp", "kind"], "moe"), "layers[0].mlp.'kind'"),
    (_edit(["layers", 3, "mixer", "kv_from"], 3), "'kv_from' = 3"),
    (_edit(["layers", 3, "mixer", "kv_from"], 0), "'kv_from' = 0"),
    (_edit(["layers", 6, "mixer", "kv_from"], 3), "'kv_from' = 3"),
    (_edit(["layers", 6, "mixer", "kv_from"], 4), "'kv_rank' differs"),
    (_edit(["layers", 3, "mixer", "rot", "base"], 7.0), "'rot' differs"),
])
def test_configuration_errors_name_the_key(edit, text):
    cfg = copy.deepcopy(MIXED)
    edit(cfg)
    with pytest.raises(ConfigError) as e:
        spec_from_config(cfg)
    assert text in str(e.value), str(e.value)


def test_absent_parts_of_the_configuration():
    cfg = copy.deepcopy(MIXED)
    for layer in cfg["layers"]:
        for key in ("rot", "mask", "softcap", "kv_heads", "kv_from"):
            layer["mixer"].pop(key, None)
        if layer["type"] == "attention":
            layer["mixer"].pop("vdim")
        layer.pop("mlp")
    _, spec = spec_from_config(cfg)
    for layer, l in zip(spec.layers, cfg["layers"]):
        assert layer.mixer["window"] == 0 and layer.mixer["position"].kind == "none" and layer.feed_forward is None
        if l["type"] == "attention":
            assert layer.mixer["num_kv_heads"] == l["mixer"]["heads"] and layer.mixer["logit_softcap"] == 0.0
    assert all(e.cache_of is None for e in spec.schedule)
    assert "l0.norm2" in spec.tolerated and "l0.norm2.b" in spec.tolerated


def test_sizes_that_the_configuration_omits_come_from_the_tensors():
    from strata_inference_b200.config.simetar import simetar_sizes
    for cfg in (MIXED, ODD):
        shapes = {n: tuple(t.shape) for n, t in random_weights(cfg, seed=1).items()}
        bare = copy.deepcopy(cfg)
        del bare["vocab"], bare["width"]
        for layer in bare["layers"]:
            for key in ("dim", "vdim", "kv_heads", "conv", "kv_rank", "rot_dim"):
                layer["mixer"].pop(key, None)
            if layer["mlp"]:
                layer["mlp"].pop("ff")
        assert spec_from_config(bare, shapes)[1] == spec_from_config(cfg)[1]
        assert simetar_sizes(cfg, shapes) == cfg


def test_rows_worked_on_whole_refuse_what_they_do_not_take():
    from strata_inference_b200.parts.attention import Attention
    _, spec = spec_from_config(ALONE["window"])
    base = dict(spec.layers[0].mixer.params)
    for extra in ({"head_temp": True}, {"value_mix": "first"}, {"pool": 8}, {"head_gate": True}, {"borrows_cache": True},
                  {"value_dim": 24}):
        with pytest.raises(ConfigError):
            Attention.tensors(dict(base, **extra), 64)


# ---- the plain model's mechanisms -----------------------------------------

def test_plain_convolution():
    rng = np.random.default_rng(0)
    h, w = rng.normal(size=(6, 3)), rng.normal(size=(3, 4))
    got = plain.causal_conv(h, w)
    assert np.allclose(got[0], w[:, 3] * h[0])
    assert np.allclose(got[2], w[:, 3] * h[2] + w[:, 2] * h[1] + w[:, 1] * h[0])
    for c in range(3):       # numpy's convolution of the channel with the reversed taps
        assert np.allclose(got[:, c], np.convolve(h[:, c], w[c, ::-1])[:6])
    assert np.allclose(plain.causal_conv(h, w[:, :1]), h * w[:, 0])
    assert np.allclose(plain.causal_conv(h[:2], w), got[:2])        # fewer rows than taps


def test_plain_layer_norm():
    rng = np.random.default_rng(1)
    x = rng.normal(size=(3, 8)) + 5.0
    y = plain.layer_norm(x, np.ones(8), np.zeros(8), 0.0)
    assert np.allclose(y.mean(-1), 0.0) and np.allclose(y.std(-1), 1.0)
    w, b = rng.normal(size=8), rng.normal(size=8)
    assert np.allclose(plain.layer_norm(x, w, b, 0.0), y * w + b)
    assert np.allclose(plain.layer_norm(np.full((1, 8), 3.0), w, b, 1e-6), b)


def test_plain_llama3_frequencies():
    dims, base, sc = 64, 10000.0, llama3(8.0, 1.0, 4.0, 1000)
    f, g = np.array(plain.plain_frequencies(dims, base)), np.array(plain.llama3_frequencies(dims, base, sc))
    turns = 1000 * f / (2 * math.pi)
    ratio = g / f
    assert (ratio[turns > 4.0] == 1.0).all() and np.allclose(ratio[turns < 1.0], 1 / 8.0)
    mid = (turns > 1.0) & (turns < 4.0)
    assert mid.any() and ((ratio[mid] > 1 / 8.0) & (ratio[mid] < 1.0)).all() and (np.diff(ratio) <= 1e-12).all()
    # a pair that makes exactly `low` turns gets f / factor from either branch, one of `high` turns f
    share = (turns[mid] - 1.0) / 3.0
    assert np.allclose(ratio[mid], (1 - share) / 8.0 + share)


def test_plain_frequencies_are_the_position_parts():
    """(the part's arithmetic is 64-bit on the CPU up to the last rounding)"""
    from strata_inference_b200.parts.position import llama3 as part_llama3, yarn as part_yarn
    for dims, base, sc in ((32, 10000.0, yarn()), (12, 500.0, yarn(3.0, 40, 5.0, 0.4)), (64, 1e6, yarn(40.0, 4096, 32.0, 1.0))):
        f = torch.tensor(plain.plain_frequencies(dims, base), dtype=torch.float64)
        got, mag = part_yarn(f, dims, base, sc)
        want, want_mag = plain.yarn_frequencies(dims, base, sc)
        assert np.allclose(got.numpy(), want, rtol=1e-13) and abs(mag - want_mag) < 1e-15
    for dims, base, sc in ((32, 10000.0, llama3()), (12, 500.0, llama3(3.0, 0.4, 5.0, 40)), (64, 1e6, llama3(40.0, 1.0, 4.0, 8192)),
                           (6, 100.0, llama3(2.0, 2.0, 2.0, 30)), (8, 10.0, llama3(5.0, 1.0, 4.0, 10 ** 6))):
        f = torch.tensor(plain.plain_frequencies(dims, base), dtype=torch.float64)
        assert np.allclose(part_llama3(f, sc).numpy(), plain.llama3_frequencies(dims, base, sc), rtol=1e-13)


def test_plain_rotations():
    rng = np.random.default_rng(2)
    x = rng.normal(size=(5, 2, 10))
    a = plain.rotate_neighbours(x, {"dims": 6, "base": 100.0})
    b = plain.rotate_halves(x, {"dims": 6, "base": 100.0})
    assert np.array_equal(a[..., 6:], x[..., 6:]) and np.array_equal(a[0], x[0]) and np.array_equal(b[0], x[0])
    for i in range(3):
        f = 100.0 ** (-2 * i / 6)
        z = (x[3, 0, 2 * i] + 1j * x[3, 0, 2 * i + 1]) * np.exp(3j * f)
        assert np.allclose([a[3, 0, 2 * i], a[3, 0, 2 * i + 1]], [z.real, z.imag])
        z = (x[3, 0, i] + 1j * x[3, 0, i + 3]) * np.exp(3j * f)
        assert np.allclose([b[3, 0, i], b[3, 0, i + 3]], [z.real, z.imag])
    c = plain.rotate_halves(x, {"dims": 6, "base": 100.0, "scaling": yarn(4.0, 50)})
    assert np.allclose(c[0, :, :6], (0.1 * math.log(4.0) + 1.0) * x[0, :, :6])


def test_plain_softmax_beside_one():
    s = np.array([0.3, -2.0, 1.5])
    assert np.allclose(plain.weights_beside_one(s), np.exp(s) / (1.0 + np.exp(s).sum()))
    assert np.allclose(plain.weights_beside_one(np.array([800.0, 0.0])), [1.0, 0.0])
    assert plain.weights_beside_one(np.array([-800.0])).max() == 0.0
    assert np.allclose(plain.softcap(s, 2.0), 2.0 * np.tanh(s / 2.0)) and plain.softcap(s, 0) is s
    assert plain.first_visible(10, 3) == 8 and plain.first_visible(1, 3) == 0 and plain.first_visible(9, 0) == 0


def test_plain_attention_by_hand():
    rng = np.random.default_rng(3)
    m = {"heads": 2, "kv_heads": 1, "dim": 4, "scale": 0.5, "softcap": 3.0, "mask": {"size": 2}}
    w = {n: rng.normal(size=s) for n, s in (("q", (8, 6)), ("k", (4, 6)), ("q.b", (8,)), ("k.b", (4,)), ("q.conv", (8, 2)),
                                            ("k.conv", (4, 2)), ("q.norm", (8,)), ("k.norm", (4,)), ("g", (8, 6)))}
    w["o"] = np.eye(8)
    h = rng.normal(size=(5, 6))
    y = plain.attention(h, w, m, 1e-6)
    uq, uk = h @ w["q"].T + w["q.b"], h @ w["k"].T + w["k.b"]
    cq = {t: w["q.conv"][:, 1] * uq[t] + w["q.conv"][:, 0] * uq[t - 1] for t in (3, 4)}
    ck = {t: w["k.conv"][:, 1] * uk[t] + w["k.conv"][:, 0] * uk[t - 1] for t in (3, 4)}
    q = cq[4] / np.sqrt((cq[4] ** 2).mean() + 1e-6) * w["q.norm"]       # (one root mean square for both heads)
    k = {t: ck[t] / np.sqrt((ck[t] ** 2).mean() + 1e-6) * w["k.norm"] for t in (3, 4)}
    for a in range(2):
        e = np.exp([3.0 * np.tanh(q[4 * a:4 * a + 4] @ k[t] * 0.5 / 3.0) for t in (3, 4)])
        o = (e[0] * ck[3] + e[1] * ck[4]) / (1.0 + e.sum())
        assert np.allclose(y[4, 4 * a:4 * a + 4], o / (1.0 + np.exp(-(h[4] @ w["g"].T)))[4 * a:4 * a + 4])


def test_plain_latent_attention_by_hand():
    rng = np.random.default_rng(4)
    m = {"heads": 2, "dim": 3, "rot_dim": 2, "vdim": 4, "kv_rank": 5, "scale": 0.7, "rot": {"dims": 2, "base": 10.0}}
    w = {n: rng.normal(size=s) for n, s in (("q", (10, 6)), ("dkv", (7, 6)), ("dkv.norm", (5,)), ("uk", (6, 5)), ("uv", (8, 5)),
                                            ("g", (8, 6)))}
    w["o"] = np.eye(8)
    h = rng.normal(size=(3, 6))
    c, shared = plain.latent_rows(h, w, m, 1e-6)
    y = plain.latent_attention(h, w, m, (c, shared))
    down = h @ w["dkv"].T
    assert np.allclose(c, down[:, :5] / np.sqrt((down[:, :5] ** 2).mean(-1, keepdims=True) + 1e-6) * w["dkv.norm"])
    turn = lambda v, p: np.array([v[0] * math.cos(p) - v[1] * math.sin(p), v[1] * math.cos(p) + v[0] * math.sin(p)])  # noqa: E731
    assert np.allclose(shared[2], turn(down[2, 5:], 2))
    for a in range(2):
        q = (w["q"] @ h[2])[5 * a:5 * a + 5]
        s = np.array([(q[:3] @ (w["uk"][3 * a:3 * a + 3] @ c[j]) + turn(q[3:], 2) @ shared[j]) * 0.7 for j in range(3)])
        p = np.exp(s) / np.exp(s).sum()
        o = sum(p[j] * (w["uv"][4 * a:4 * a + 4] @ c[j]) for j in range(3))
        assert np.allclose(y[2, 4 * a:4 * a + 4], o / (1.0 + np.exp(-(w["g"] @ h[2])[4 * a:4 * a + 4])))


def test_plain_layer_norms_what_it_adds():
    cfg = model(16, 20, [attention(2, 1, 4, 3, mlp=dense(8)), latent(1, 4, 2, 4, 6), latent(2, 4, 2, 4, 6, kv_from=1)])
    w = random_weights(cfg, seed=5)
    toks = [1, 2, 3, 4, 5]
    x0 = plain.f64(w["embed"])[toks]
    n = lambda x, name: plain.layer_norm(x, plain.f64(w[name]), plain.f64(w[name + ".b"]), 1e-5)  # noqa: E731
    x1 = x0 + n(plain.attention(x0, plain.sub(w, "l0.mix."), cfg["layers"][0]["mixer"], 1e-5), "l0.norm1")
    ff = plain.sub(w, "l0.mlp.")
    z = x1 @ ff["gate"].T
    act = 0.5 * z * (1 + np.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))
    x2 = x1 + n((act * (x1 @ ff["up"].T)) @ ff["down"].T, "l0.norm2")
    m1, m2 = cfg["layers"][1]["mixer"], cfg["layers"][2]["mixer"]
    kept = plain.latent_rows(x2, plain.sub(w, "l1.mix."), m1, 1e-5)
    x3 = x2 + n(plain.latent_attention(x2, plain.sub(w, "l1.mix."), m1, kept), "l1.norm1")
    x4 = x3 + n(plain.latent_attention(x3, plain.sub(w, "l2.mix."), m2, kept), "l2.norm1")
    streams = plain.layer_streams(cfg, w, toks)
    assert np.allclose(streams[0], x2) and np.allclose(streams[1], x3) and np.allclose(streams[2], x4)
    assert np.allclose(plain.logits(cfg, w, toks), n(x4, "final.norm") @ plain.f64(w["head"]).T)
