"""Kerolorn on the CPU: the configuration and its layout as parts, the cache's cells of kept first
positions, and the plain model's own mechanisms (tests/plain_kerolorn.py) against closed forms."""

from __future__ import annotations

import copy
import math

import numpy as np
import pytest
import torch

import plain_kerolorn as plain
from kerolorn_cases import ALONE, MIXED, ODD, WIDE, attention, model, moe, random_weights, yarn

from strata_inference_b200.cache.paged import CacheError, CacheNeed, KVNeed, SequenceCache, StateNeed
from strata_inference_b200.config.registry import spec_from_config
from strata_inference_b200.config.spec import ConfigError
from strata_inference_b200.engine.model import expected_tensors


def test_every_size_and_constant_comes_from_the_configuration():
    typed, spec = spec_from_config(MIXED)
    assert spec.architecture == "Kerolorn" and spec.hidden_size == 64 and spec.vocab_size == 200
    assert spec.head["logit_scale"] == 0.5 and not spec.head["tied"]
    first, second, last = spec.layers[0], spec.layers[1], spec.layers[4]
    assert first.block == "sandwich" and first.mixer_input.kind == "short_conv" and first.mixer_input["taps"] == 4
    m = first.mixer
    assert (m["num_heads"], m["num_kv_heads"], m["head_dim"], m["value_dim"]) == (4, 2, 16, 16)
    assert (m["window"], m["keep_first"], m["score_scale"]) == (37, 12, 0.2)
    assert m["head_temp"] and m["qk_norm"] == {"eps": 1e-5, "weight": False, "after_rotation": True}
    assert m["position"].kind == "rope_interleaved" and m["position"]["rotary_dim"] == 8
    assert m["position"]["yarn"] == yarn()
    assert second.mixer["value_dim"] == 48 and second.mixer["position"]["yarn"] is None
    assert spec.layers[2].mixer["window"] == 0 and spec.layers[2].mixer["keep_first"] == 0
    assert spec.layers[3].feed_forward is None and "post_feed_forward" not in spec.layers[3].norms
    assert last.mixer["position"].kind == "none"
    ff = first.feed_forward
    assert ff.kind == "routed_experts" and (ff["experts"], ff["top"], ff["intermediate_size"]) == (6, 2, 24)
    assert (ff["form"], ff["score"], ff["correction"], ff["router_scale"]) == ("gated_silu", "softmax_all", True, 1.7)
    assert ff["shared"] == {"intermediate_size": 32, "gate": True} and second.feed_forward["shared"] is None
    assert {s: n["eps"] for s, n in first.norms.items()} == dict.fromkeys(
        ("pre_mixer", "post_mixer", "pre_feed_forward", "post_feed_forward"), 1e-5)


@pytest.mark.parametrize("cfg", [MIXED, ODD, WIDE] + [ALONE[k] for k in sorted(ALONE)])
def test_tensor_table_matches_the_random_weights(cfg):
    _, spec = spec_from_config(cfg)
    table = expected_tensors(spec)
    w = random_weights(cfg, seed=1)
    needed = {n for n, d in table.items() if not d.optional}
    assert needed == set(w), (sorted(needed - set(w)), sorted(set(w) - needed))
    for n in needed:
        assert tuple(table[n].shape) == tuple(w[n].shape), n


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
    (_edit(["logit_scale"], None), "logit_scale"),
    (_edit(["canon"], None), "canon"),
    (_edit(["canon", "taps"], 0), "canon.'taps'"),
    (_edit(["layers", 0, "type"], "recurrent"), "layers[0].'type'"),
    (_edit(["layers", 0, "mixer", "scale"], "x"), "layers[0].mixer.'scale'"),
    (_edit(["layers", 0, "mixer", "kv_heads"], 3), "kv_heads"),
    (_edit(["layers", 0, "mixer", "rot", "dims"], 7), "layers[0].mixer.rot"),
    (_edit(["layers", 0, "mixer", "rot", "scaling", "slow"], None), "layers[0].mixer.rot.scaling.'slow'"),
    (_edit(["layers", 0, "mixer", "mask", "size"], 0), "layers[0].mixer.mask.'size'"),
    (_edit(["layers", 0, "mixer", "mask", "keep_first"], -1), "layers[0].mixer.mask.'keep_first'"),
    (_edit(["layers", 0, "mlp", "kind"], "dense"), "layers[0].mlp.'kind'"),
    (_edit(["layers", 0, "mlp", "router", "top"], 9), "'top' exceeds 'experts'"),
    (_edit(["layers", 0, "mlp", "expert"], None), "layers[0].mlp.'expert'"),
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
        layer["mixer"].pop("rot", None)
        layer["mixer"].pop("mask", None)
        layer["mixer"].pop("kv_heads")
        layer.pop("mlp")
    _, spec = spec_from_config(cfg)
    for layer, l in zip(spec.layers, cfg["layers"]):
        assert layer.mixer["window"] == 0 and layer.mixer["position"].kind == "none" and layer.feed_forward is None
        assert layer.mixer["num_kv_heads"] == l["mixer"]["heads"]
    assert "l0.norm2" in spec.tolerated and "l0.norm2b" in spec.tolerated


def test_sizes_that_the_configuration_omits_come_from_the_tensors():
    from strata_inference_b200.config.kerolorn import kerolorn_sizes
    for cfg in (MIXED, ODD):
        shapes = {n: tuple(t.shape) for n, t in random_weights(cfg, seed=1).items()}
        bare = copy.deepcopy(cfg)
        del bare["vocab"], bare["width"], bare["canon"]
        for layer in bare["layers"]:
            for key in ("heads", "dim", "vdim", "kv_heads"):
                layer["mixer"].pop(key)
            if layer["mlp"]:
                layer["mlp"]["router"].pop("experts")
                layer["mlp"]["expert"].pop("ff")
                if layer["mlp"].get("shared"):
                    layer["mlp"]["shared"].pop("ff")
        assert spec_from_config(bare, shapes)[1] == spec_from_config(cfg)[1]
        assert kerolorn_sizes(cfg, shapes) == cfg


def _cache(window, keep, max_seq_len=1024, **kw):
    needs = [CacheNeed(kv=KVNeed(1, 16, window, keep_first=keep), inputs=StateNeed((12,)))]
    return SequenceCache(needs, 4096, max_seq_len, torch.float32, "cpu", page_tokens=16, max_slots=3, **kw)


def test_kept_first_positions_have_pages_of_their_own_ahead_of_the_ring():
    c = _cache(40, 20)
    g = c.groups[0]
    assert g.fixed_tokens == 32 and g.ring_tokens == 64 and g.pages_per_seq == 6
    v = c.kv_view(0)
    assert (v.fixed_tokens, v.ring_tokens) == (32, 64)
    # a step may add what leaves the keys its first row still sees where they are
    assert g.max_step_tokens() == 25 and g.max_step_tokens(10) == 86 and g.max_step_tokens(90) == 25
    s = c.acquire()
    for n, pages in ((1, 1), (31, 2), (1, 3), (63, 6), (500, 6)):
        c.reserve([(s, n)])
        c.advance(s, n)
        assert len(g.pages[s]) == pages
    assert len(set(g.pages[s])) == 6
    # every position that a later one may see has a cell that nothing else in sight occupies
    for end in range(1, 300):
        seen = [p for p in range(end) if end - 1 - p < 40 or p < 20]
        cells = [p if p < g.fixed_tokens else g.fixed_tokens + (p - g.fixed_tokens) % g.ring_tokens for p in seen]
        assert len(set(cells)) == len(cells)
    c.release(s)
    assert g.pool.n_free == g.n_pages


def test_a_window_and_kept_positions_that_reach_the_whole_length_need_no_ring():
    g = _cache(40, 20, max_seq_len=96).groups[0]
    assert g.ring_tokens == 0 and g.fixed_tokens == 0 and g.pages_per_seq == 6
    assert _cache(40, 0).groups[0].fixed_tokens == 0
    with pytest.raises(CacheError):
        _cache(0, 5)


def test_the_state_at_a_mixers_input_is_zeroed_when_a_slot_is_taken():
    c = _cache(40, 20)
    s = c.acquire()
    c.input_state_view(0)[s] = 7.0
    c.release(s)
    assert c.acquire() == s and float(c.input_state_view(0)[s].abs().sum()) == 0.0
    assert 0 not in c.state


def test_plain_convolution():
    rng = np.random.default_rng(0)
    h, w = rng.normal(size=(6, 3)), rng.normal(size=(3, 4))
    got = plain.causal_conv(h, w)
    assert np.allclose(got[0], w[:, 3] * h[0])
    assert np.allclose(got[2], w[:, 3] * h[2] + w[:, 2] * h[1] + w[:, 1] * h[0])
    for c in range(3):       # numpy's convolution of the channel with the reversed taps
        assert np.allclose(got[:, c], np.convolve(h[:, c], w[c, ::-1])[:6])
    assert np.allclose(plain.causal_conv(h, w[:, :1]), h * w[:, 0])


def test_plain_yarn_frequencies():
    dims, base = 32, 10000.0
    freqs, mag = plain.yarn_frequencies(dims, base, None)
    assert mag == 1.0 and np.allclose(freqs, [base ** (-2 * i / dims) for i in range(16)])
    sc = yarn(8.0, 1000, 32.0, 1.0)
    slow, mag = plain.yarn_frequencies(dims, base, sc)
    assert abs(mag - (0.1 * math.log(8.0) + 1.0)) < 1e-12
    # the fastest pair keeps its frequency, the slowest is divided by the factor, the ratio falls in between
    ratio = np.array(slow) / np.array(freqs)
    assert ratio[0] == 1.0 and abs(ratio[-1] - 1 / 8.0) < 1e-12 and (np.diff(ratio) <= 1e-12).all()
    # at the (real) index of `turns`, the plain frequency makes that many turns in `original` positions
    idx = dims * math.log(1000 / (2 * math.pi * 32.0)) / (2 * math.log(base))
    assert abs(base ** (-2 * idx / dims) * 1000 - 2 * math.pi * 32.0) < 1e-9
    lo, hi = math.floor(idx), math.ceil(dims * math.log(1000 / (2 * math.pi)) / (2 * math.log(base)))
    assert ratio[lo] == 1.0 and abs(ratio[hi] - 1 / 8.0) < 1e-12 and 1 / 8.0 < ratio[(lo + hi) // 2] < 1.0


def test_plain_frequencies_are_the_position_parts():
    """(the part's arithmetic is 64-bit on the CPU up to the last rounding)"""
    from strata_inference_b200.parts.position import yarn as part_yarn
    for dims, base, sc in ((32, 10000.0, yarn()), (12, 500.0, yarn(3.0, 40, 5.0, 0.4)), (64, 1e6, yarn(40.0, 4096, 32.0, 1.0)),
                           (6, 100.0, yarn(2.0, 10, 100.0, 50.0)), (8, 10.0, yarn(4.0, 10 ** 6, 2.0, 1.0))):
        plain_f = torch.tensor(plain.yarn_frequencies(dims, base, None)[0], dtype=torch.float64)
        got, mag = part_yarn(plain_f, dims, base, sc)
        want, want_mag = plain.yarn_frequencies(dims, base, sc)
        assert np.allclose(got.numpy(), want, rtol=1e-13) and abs(mag - want_mag) < 1e-15


def test_plain_rotation_then_norm():
    rng = np.random.default_rng(1)
    x = rng.normal(size=(4, 2, 10))
    y = plain.rotate_pairs(x, [0, 1, 5, 300], 6, [1.0, 0.1, 0.01], 1.25)
    assert np.array_equal(y[..., 6:], x[..., 6:]) and np.allclose(y[0, :, :6], 1.25 * x[0, :, :6])
    for i in range(3):
        assert np.allclose(np.hypot(y[..., 2 * i], y[..., 2 * i + 1]), 1.25 * np.hypot(x[..., 2 * i], x[..., 2 * i + 1]))
    u = plain.unit_rms(y, 0.0)
    assert np.allclose((u ** 2).mean(-1), 1.0)
    # (with a magnitude and a part that is not rotated, norming before the rotation is another function)
    v = plain.rotate_pairs(plain.unit_rms(x, 0.0), [0, 1, 5, 300], 6, [1.0, 0.1, 0.01], 1.25)
    assert not np.allclose(u, v)


def test_plain_mask_and_head_factors():
    assert plain.visible(10, 3, 2) == [0, 1, 8, 9, 10] and plain.visible(3, 3, 2) == [0, 1, 2, 3]
    assert plain.visible(2, 3, 9) == [0, 1, 2] and plain.visible(12, 3, 9) == list(range(9)) + [10, 11, 12]
    assert plain.visible(5, 0, 0) == list(range(6)) and plain.visible(9, 1, 0) == [9]
    rng = np.random.default_rng(2)
    m = {"heads": 2, "kv_heads": 1, "dim": 4, "vdim": 3, "scale": 0.5, "mask": {"size": 2, "keep_first": 1}}
    w = {"q": rng.normal(size=(8, 6)), "k": rng.normal(size=(4, 6)), "v": rng.normal(size=(3, 6)), "o": np.eye(6),
         "temp": np.array([0.0, 3.0])}
    h = rng.normal(size=(5, 6))
    y = plain.attention(h, w, m, 1e-6)
    v = h @ w["v"].T
    assert np.allclose(y[4, :3], (v[0] + v[3] + v[4]) / 3)        # a head whose factor is 0 averages
    q, k = plain.unit_rms(h @ w["q"][4:].T, 1e-6), plain.unit_rms(h @ w["k"].T, 1e-6)
    s = np.exp(np.array([q[4] @ k[j] for j in (0, 3, 4)]) * 0.5 * 3.0)
    assert np.allclose(y[4, 3:], (s / s.sum()) @ v[[0, 3, 4]])


def test_plain_experts():
    rng = np.random.default_rng(3)
    mlp = moe(3, 2, 4, shared=2, scale=2.0)
    w = {"router": np.eye(3, 6), "correction": np.array([0.0, 0.9, 0.0]), "shared.sg": rng.normal(size=(1, 6))}
    for n, f in (("e0", 4), ("e1", 4), ("e2", 4), ("shared", 2)):
        w[n + ".gate"], w[n + ".up"], w[n + ".down"] = rng.normal(size=(f, 6)), rng.normal(size=(f, 6)), rng.normal(size=(6, f))
    x = np.array([[2.0, -1.0, 0.5, 0.3, 0.1, -0.2]])
    ids, ps = plain.router_choice(x, w, mlp)
    s = np.exp(x[0, :3]) / np.exp(x[0, :3]).sum()
    assert ids[0].tolist() == [1, 0]          # the correction lifts the smallest score to the first place
    assert np.allclose(ps[0], 2.0 * s[[1, 0]])  # and does not enter the weight; nothing is normalized

    def one(n):
        g = x @ w[n + ".gate"].T
        return (g / (1 + np.exp(-g)) * (x @ w[n + ".up"].T)) @ w[n + ".down"].T
    want = 2.0 * (s[1] * one("e1") + s[0] * one("e0")) + one("shared") / (1 + np.exp(-(x @ w["shared.sg"].T)))
    assert np.allclose(plain.routed_ff(x, w, mlp), want)


def test_plain_layer_norms_what_it_adds():
    cfg = model(16, 20, [attention(2, 1, 4, 4, 3, 1, mlp=moe(2, 1, 8))], taps=2)
    w = random_weights(cfg, seed=5)
    toks = [1, 2, 3, 4, 5]
    x0 = plain.f64(w["embed"])[toks]
    n = lambda x, name: x / np.sqrt((x * x).mean(-1, keepdims=True) + 1e-5) * plain.f64(w[name])  # noqa: E731
    h = n(x0, "l0.norm1")
    c = plain.f64(w["l0.canon1"])
    h = h + c[:, 1] * h + c[:, 0] * np.vstack([np.zeros(16), h[:-1]])
    x1 = x0 + n(plain.attention(h, plain.sub(w, "l0.mix."), cfg["layers"][0]["mixer"], 1e-5), "l0.norm1b")
    x2 = x1 + n(plain.routed_ff(n(x1, "l0.norm2"), plain.sub(w, "l0.mlp."), cfg["layers"][0]["mlp"]), "l0.norm2b")
    assert np.allclose(plain.layer_streams(cfg, w, toks)[0], x2)
    assert np.allclose(plain.logits(cfg, w, toks), 0.5 * n(x2, "final.norm") @ plain.f64(w["head"]).T)
