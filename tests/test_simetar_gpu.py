"""Simetar through the engine against the plain model (tests/plain_simetar.py): each mechanism alone,
prompts against token-by-token steps, portions, unequal batches, slots and pages used again, the
edges of windows and far keys with a softmax that picks single keys, the added one of the softmax,
lent rows, the first tokens of a sequence, long decoding, odd and wide sizes, configurations drawn
at random, the kernels alone, greedy generation and trace replay."""

from __future__ import annotations

import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_simetar as plain
from simetar_cases import (ALONE, MIXED, ODD, SHARP, WIDE, assert_close, attention, changed, dense, latent, llama3, model,
                           plain_logits, prompts, random_model, random_weights, rows_that_differ, yarn)

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def make_engine(cfg, weights, dtype, **kw):
    from strata_inference_b200.config.registry import spec_from_config
    from strata_inference_b200.engine.engine import Engine
    _, spec = spec_from_config(cfg)
    kw.setdefault("max_tokens", 2048)
    kw.setdefault("max_seq_len", 1024)
    return Engine(spec, weights, dtype=dtype, **kw)


def all_rows(n):
    return list(range(n))


def run_whole(eng, tokens):
    s = eng.new_sequence()
    out = eng.step([(s, tokens)], [all_rows(len(tokens))])
    eng.end_sequence(s)
    return out


def run_portions(eng, tokens, sizes):
    """The prompt cut into steps of the given sizes (the last takes the rest)."""
    s, at, rows = eng.new_sequence(), 0, []
    for n in list(sizes) + [len(tokens)]:
        part = tokens[at:at + n]
        if not part:
            break
        rows.append(eng.step([(s, part)], [all_rows(len(part))]))
        at += len(part)
    eng.end_sequence(s)
    return torch.cat(rows)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ALONE))
def test_each_mechanism_alone(name, dtype):
    cfg = ALONE[name]
    w = random_weights(cfg, 11)
    eng = make_engine(cfg, w, dtype)
    for toks in prompts(cfg, [1, 2, 5, 90], seed=3):
        assert_close(run_whole(eng, toks), plain_logits(cfg, w, toks), dtype, f"{name}, {len(toks)} tokens")
    toks = prompts(cfg, [130], seed=4)[0]
    assert_close(run_portions(eng, toks, [3, 1, 1, 2, 50] + [1] * 8 + [24, 16] + [1] * 20), plain_logits(cfg, w, toks), dtype,
                 f"{name} in portions and single tokens")


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompt_then_long_decoding(dtype):
    """A prompt in one step, then 400 single-token steps (every ring wraps several times; the
    token steps are recorded at the second and replayed from the third), and token by token from
    the very first token."""
    cfg = MIXED
    w = random_weights(cfg, 5)
    eng = make_engine(cfg, w, dtype)
    toks = prompts(cfg, [440], seed=6)[0]
    ref = plain_logits(cfg, w, toks)
    assert_close(run_portions(eng, toks, [40] + [1] * 400), ref, dtype, "prompt of 40, then token by token")
    assert_close(run_portions(eng, toks[:150], [1] * 130 + [20]), ref[:150], dtype, "token by token from the first token")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[2] * 30, [64, 25], [63, 2, 24], [1, 24, 3, 23], [17, 17, 17, 17, 17], [3, 2, 4, 2, 37, 1, 36],
                                   [7, 8, 9, 16, 1, 15, 24], [36, 2, 12, 38, 2], [40, 40, 20, 39, 2], [130, 2]])
def test_portions(sizes, dtype):
    """(portions shorter and longer than the convolutions' reach, across the edges of the windows of
    37 and 90 and of pages)"""
    cfg = MIXED
    w = random_weights(cfg, 7)
    eng = make_engine(cfg, w, dtype)
    toks = prompts(cfg, [210], seed=8)[0]
    assert_close(run_portions(eng, toks, sizes + [20] * 11), plain_logits(cfg, w, toks), dtype, f"portions {sizes}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_batch_against_each_alone(dtype):
    """Prompts of 1 to 130 tokens in one step, then single-token steps together; the
    shorter requests end earlier and a new one takes a freed slot later."""
    cfg = MIXED
    w = random_weights(cfg, 9)
    eng = make_engine(cfg, w, dtype)
    reqs = prompts(cfg, [21, 22, 100, 160, 35], seed=10)
    first = [1, 2, 70, 130, 5]
    refs = [plain_logits(cfg, w, t) for t in reqs]
    live = [0, 1, 2, 3]
    slots = {i: eng.new_sequence() for i in live}
    out = eng.step([(slots[i], reqs[i][:first[i]]) for i in live], [all_rows(first[i]) for i in live])
    at = 0
    for i in live:
        assert_close(out[at:at + first[i]], refs[i][:first[i]], dtype, f"batched prompt {i}")
        at += first[i]
    pos = {i: first[i] for i in live}
    step = 0
    while live:
        if step == 25:                         # the latecomer starts alone, then decodes with the rest
            slots[4] = eng.new_sequence()
            got = eng.step([(slots[4], reqs[4][:first[4]])], [all_rows(first[4])])
            assert_close(got, refs[4][:first[4]], dtype, "late prompt")
            pos[4] = first[4]
            live.append(4)
        out = eng.step([(slots[i], [reqs[i][pos[i]]]) for i in live], [[0]] * len(live))
        for k, i in enumerate(live):
            assert_close(out[k:k + 1], refs[i][pos[i]:pos[i] + 1], dtype, f"request {i}, token {pos[i]}")
            pos[i] += 1
        for i in list(live):
            if pos[i] == len(reqs[i]):
                eng.end_sequence(slots[i])
                live.remove(i)
        step += 1
    assert step > 25


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_of_several_requests_in_one_step(dtype):
    """Steps that mix a first portion, a later portion and a single token."""
    cfg = MIXED
    w = random_weights(cfg, 19)
    eng = make_engine(cfg, w, dtype)
    reqs = prompts(cfg, [120, 90, 60], seed=20)
    refs = [plain_logits(cfg, w, t) for t in reqs]
    cuts = [[50, 2, 40, 1, 27], [0, 30, 1, 57, 2], [0, 0, 3, 55, 2]]
    slots, pos = [eng.new_sequence() for _ in reqs], [0, 0, 0]
    for k in range(5):
        live = [i for i in range(3) if cuts[i][k]]
        out = eng.step([(slots[i], reqs[i][pos[i]:pos[i] + cuts[i][k]]) for i in live], [all_rows(cuts[i][k]) for i in live])
        at = 0
        for i in live:
            n = cuts[i][k]
            assert_close(out[at:at + n], refs[i][pos[i]:pos[i] + n], dtype, f"step {k}, request {i}")
            at += n
            pos[i] += n
    assert pos == [120, 90, 60]


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_and_pages_used_again(dtype):
    """A slot that is given back and taken again starts from nothing: convolution histories and pages
    of the request before leave no trace; with few pages they are all used again."""
    cfg = MIXED
    w = random_weights(cfg, 12)
    eng = make_engine(cfg, w, dtype, max_tokens=512, max_seq_len=256, max_slots=2)
    a, b, c = prompts(cfg, [100, 90, 120], seed=13)
    ra, rb, rc = (plain_logits(cfg, w, t) for t in (a, b, c))
    sa = eng.new_sequence()
    assert_close(eng.step([(sa, a[:70])], [all_rows(70)]), ra[:70], dtype, "a, first part")
    sb = eng.new_sequence()
    assert_close(eng.step([(sb, b[:50])], [all_rows(50)]), rb[:50], dtype, "b, first part")
    assert_close(eng.step([(sa, a[70:])], [all_rows(30)]), ra[70:], dtype, "a, second part")
    eng.end_sequence(sa)
    sc = eng.new_sequence()
    assert sc == sa
    assert_close(eng.step([(sc, c[:1])], [[0]]), rc[:1], dtype, "c's first token in a's slot")
    assert_close(eng.step([(sc, c[1:110])], [all_rows(109)]), rc[1:110], dtype, "c in a's slot and pages")
    out = eng.step([(sb, [b[50]]), (sc, [c[110]])], [[0], [0]])
    assert_close(out, torch.stack([rb[50], rc[110]]), dtype, "b and c together")
    assert_close(eng.step([(sb, b[51:])], [all_rows(39)]), rb[51:], dtype, "b, the rest")
    eng.end_sequence(sb)
    eng.end_sequence(sc)
    assert_close(run_whole(eng, a), ra, dtype, "a once more")


@pytest.mark.parametrize("page_tokens", [16, 64])
def test_edges_of_windows_with_a_sharp_softmax(page_tokens):
    """With a large scale the softmax puts most of a row's weight on single keys, wherever in
    sight they lie.  The plain model with windows one shorter or one longer gives other logits in
    many rows (checked first: the test can tell them apart); the engine agrees with the right one as
    a prompt, in portions around page borders, token by token through several turns of the ring, and
    as two requests side by side."""
    cfg, dtype = SHARP, "float32"
    w = random_weights(cfg, seed=14)
    toks = prompts(cfg, [330], seed=15)[0]
    ref = plain_logits(cfg, w, toks)

    def mask(delta):
        def edit(c):
            for layer in c["layers"]:
                if "mask" in layer["mixer"]:
                    layer["mixer"]["mask"]["size"] += delta
        return edit
    for delta in (-1, 1):
        other = plain_logits(changed(cfg, mask(delta)), w, toks)
        assert rows_that_differ(ref[90:], other[90:], 20.0) > 100, f"windows off by {delta} would not show"
    eng = make_engine(cfg, w, dtype, page_tokens=page_tokens)
    assert_close(run_whole(eng, toks), ref, dtype, "whole prompt")
    n = min(eng.cache.max_step_tokens(), 64)
    assert_close(run_portions(eng, toks, [64] + [n] * 40), ref, dtype, f"portions of {n}")
    assert_close(run_portions(eng, toks, [63, 2, n - 1, 1, 1, min(16, n), n - 2] + [n] * 40), ref, dtype, "portions around page borders")
    assert_close(run_portions(eng, toks, [8, 2, 7, 1, 1, 30, 2, min(14, n), 2] + [n, 1, 2, 3] * 30), ref, dtype, "portions at the edges")
    assert_close(run_portions(eng, toks, [60] + [1] * 270), ref, dtype, "single tokens through several turns of the ring")
    a, b = toks[:250], prompts(cfg, [180], seed=16)[0]
    rb = plain_logits(cfg, w, b)
    sa, sb = eng.new_sequence(), eng.new_sequence()
    out = eng.step([(sa, a[:195]), (sb, b[:40])], [all_rows(195), all_rows(40)])
    assert_close(out, torch.cat([ref[:195], rb[:40]]), dtype, "two prompts")
    for k in range(55):
        out = eng.step([(sa, [a[195 + k]]), (sb, [b[40 + k]])], [[0], [0]])
        assert_close(out, torch.stack([ref[195 + k], rb[40 + k]]), dtype, f"two requests, token {k}")


ASKS, ASKED = 47, 46


def _asking(cfg, seed):
    """Weights with which token ASKS has token ASKED's key as its query in the last layer: its weight
    goes to where that token occurs.  Earlier layers add nothing to the stream."""
    w = random_weights(cfg, seed)
    last, pre = cfg["layers"][-1], f"l{len(cfg['layers']) - 1}.mix."
    for i in range(len(cfg["layers"]) - 1):
        w[f"l{i}.norm1"].zero_()
        w[f"l{i}.norm1.b"].zero_()
    asks, asked = w["embed"][ASKS], w["embed"][ASKED]
    m = last["mixer"]
    if last["type"] == "attention":
        for n in ("q", "k"):
            w[pre + n + ".b"].zero_()
            w[pre + n + ".conv"].zero_()
            w[pre + n + ".conv"][:, -1] = 1.0
            w[pre + n + ".norm"].fill_(1.0)
        key = w[pre + "k"] @ asked
        w[pre + "q"] = torch.outer(key, asks) / asks.dot(asks)
    else:
        src = "l%d.mix." % m.get("kv_from", len(cfg["layers"]) - 1)
        c, _ = plain.latent_rows(plain.f64(w["embed"]), plain.sub(w, src), dict(m, rot=None), cfg["norm"]["eps"])
        keys = torch.from_numpy(c) @ w[pre + "uk"].double().T
        key = torch.linalg.solve(keys.T @ keys, keys[ASKED])         # (as little as can be of the other tokens' keys)
        key = key * (24.0 / m["scale"] / key.dot(keys[ASKED]))
        q = torch.zeros_like(w[pre + "q"])
        q[:m["dim"]] = (torch.outer(key, asks.double()) / asks.double().dot(asks.double())).float()
        w[pre + "q"] = q
    return {n: t.to(torch.bfloat16).float() for n, t in w.items()}


@pytest.mark.parametrize("mode", ["prompt", "tokens", "portions"])
@pytest.mark.parametrize("size", [30, 64, 65, 128, 300])
def test_a_key_just_in_and_just_out_of_sight(size, mode):
    """The last token asks for another that occurs once.  At size - 1 positions back that is seen;
    one further it is not; the row's logits differ widely between the two (checked on the plain
    model first), in a prompt, when the asking token is decoded alone, and at the end of a portion."""
    cfg = model(32, 50, [attention(1, 1, 16, size, conv=2, scale=1.0, softcap=40.0, rot_dims=0)])
    w = _asking(cfg, 40)
    eng = make_engine(cfg, w, "float32")
    far = max(size + 150, 260)
    for start, seen in ((far - 1 - (size - 1), True), (far - 1 - size, False)):
        toks = [3 + (i % 40) for i in range(far)]
        toks[start], toks[far - 1] = ASKED, ASKS
        ref = plain_logits(cfg, w, toks)
        blind = list(toks)
        blind[start] = 45
        moved = rows_that_differ(ref[-1:], plain_logits(cfg, w, blind)[-1:], 50.0)
        assert moved == (1 if seen else 0), (start, seen)
        sizes = {"prompt": [far], "tokens": [far - 25] + [1] * 25, "portions": [far - 100] + [20] * 5}[mode]
        assert_close(run_portions(eng, toks, sizes), ref, "float32", f"window {size}, key at {start} ({mode})")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("lent", [False, True])
def test_a_far_key_of_the_latent_attention(lent, dtype):
    """One key among several hundred, at the first position, at both sides of page borders and just
    before the asking token, read from the layer's own rows or from a lender's."""
    layers = [latent(1, 16, 4, 16, 20, scale=2.0)]
    if lent:
        layers = [latent(2, 8, 4, 8, 20), latent(1, 16, 4, 16, 20, scale=2.0, kv_from=0)]
    cfg = model(32, 50, layers)
    w = _asking(cfg, 41)
    eng = make_engine(cfg, w, dtype)
    for start in (0, 63, 64, 127, 128, 300, 458):
        toks = [3 + (i % 40) for i in range(460)]
        toks[start], toks[-1] = ASKED, ASKS
        ref = plain_logits(cfg, w, toks)
        blind = list(toks)
        blind[start] = 45
        assert rows_that_differ(ref[-1:], plain_logits(cfg, w, blind)[-1:], 500.0) == 1
        for sizes in ([460], [459, 1], [300, 100, 58, 2], [435] + [1] * 25):
            assert_close(run_portions(eng, toks, sizes)[-1:], ref[-1:], dtype, f"key at {start}, steps {sizes[:4]}")


def test_the_added_one_the_cap_and_the_gate_show():
    """Plain models without the added one, without the cap, with a norm per head, or without the gate
    or the slowed-down frequencies give other logits in nearly every row; the engine agrees with the
    right one, a sequence's first rows (where the added one weighs most) included."""
    cfg, dtype = model(64, 200, [attention(4, 2, 16, 60, conv=2, scale=0.5, softcap=2.0, rot_dims=6, scaling=llama3())]), "float32"
    w = random_weights(cfg, seed=26)
    toks = prompts(cfg, [150], seed=27)[0]
    ref = plain_logits(cfg, w, toks)

    def differs(name, other):
        keep = getattr(plain, name)
        setattr(plain, name, other)
        try:
            return rows_that_differ(ref, plain_logits(cfg, w, toks), 10.0)
        finally:
            setattr(plain, name, keep)
    # (far into a window the one is little beside the sum, and much of a common factor goes in the norm)
    assert differs("weights_beside_one", plain.softmax) > 70
    assert differs("softcap", lambda s, cap: s) > 130
    assert differs("sigmoid", lambda z: np.ones_like(z)) > 140
    assert differs("llama3_frequencies", lambda d, b, s: plain.plain_frequencies(d, b)) > 100
    norm = plain.rms_norm
    assert differs("rms_norm", lambda x, g, eps: (norm(x.reshape(len(x), -1, 16), 1.0, eps)).reshape(x.shape) * g) > 140
    eng = make_engine(cfg, w, dtype)
    assert_close(run_whole(eng, toks), ref, dtype, "whole prompt")
    assert_close(run_portions(eng, toks, [1] * 10 + [60, 2] + [1] * 78), ref, dtype, "portions and single tokens")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [16, 64])
def test_a_sink_above_all_scores(dim, dtype):
    """Where every score is far below 0 the added one takes nearly all of the weight (here scores lie
    near -11): what is left is summed against it in every kernel."""
    cfg = model(64, 100, [attention(2, 1, dim, 50, conv=1, scale=12.0 / dim, softcap=30.0, rot_dims=0)])
    w = random_weights(cfg, seed=30)
    w["l0.mix.q"], w["l0.mix.k"] = 0.3 * w["l0.mix.q"], 0.3 * w["l0.mix.k"]
    w["l0.mix.q.b"], w["l0.mix.k.b"] = torch.ones(2 * dim), -torch.ones(dim)        # (opposite directions)
    for n in ("q", "k"):
        w[f"l0.mix.{n}.conv"].fill_(1.0)
        w[f"l0.mix.{n}.norm"].fill_(1.0)
    w["l0.mix.k.conv"].fill_(64.0)        # (values that are large, so that what is left shows)
    w = {n: t.to(torch.bfloat16).float() for n, t in w.items()}
    toks = prompts(cfg, [200], seed=31)[0]
    ref = plain_logits(cfg, w, toks)
    keep = plain.weights_beside_one
    plain.weights_beside_one = lambda s: np.exp(s)           # the added one alone
    try:
        alone = plain_logits(cfg, w, toks)
    finally:
        plain.weights_beside_one = keep
    assert (alone - ref).abs().max() < 0.2 * ref.abs().max()
    eng = make_engine(cfg, w, dtype)
    for sizes in ([200], [100, 40, 60], [190] + [1] * 10):
        assert_close(run_portions(eng, toks, sizes), ref, dtype, f"heads of {dim}, {sizes[:3]}")


def test_lent_rows():
    """A reader of another layer's rows differs from one that makes its own; lenders are told apart
    (the plain model with the readers exchanged gives other logits)."""
    cfg = model(64, 120, [latent(2, 16, 8, 16, 24, scaling=yarn(), mlp=dense(32)), latent(3, 16, 8, 8, 24, scaling=yarn()),
                          latent(4, 8, 8, 24, 24, scaling=yarn(), kv_from=0), latent(1, 16, 8, 8, 24, scaling=yarn(), kv_from=1),
                          latent(2, 24, 8, 16, 24, scaling=yarn(), kv_from=0)])
    w = random_weights(cfg, seed=28)
    toks = prompts(cfg, [170], seed=29)[0]
    ref = plain_logits(cfg, w, toks)

    def swap(c):
        c["layers"][2]["mixer"]["kv_from"], c["layers"][3]["mixer"]["kv_from"] = 1, 0
    assert rows_that_differ(ref, plain_logits(changed(cfg, swap), w, toks), 50.0) > 160
    for dtype in DTYPES:
        eng = make_engine(cfg, w, dtype)
        assert len(eng.cache.groups) == 1 and len(eng.cache.groups[0].entries) == 2, "readers keep no rows of their own"
        for sizes in ([170], [100, 2, 30, 20] + [1] * 18, [1] * 40 + [130]):
            assert_close(run_portions(eng, toks, sizes), ref, dtype, f"portions {sizes[:5]}")


def test_the_convolutions_reach():
    """The last taps - 1 projected rows of a sequence are carried from step to step in every attention
    layer: a plain model that forgets them differs in the rows behind."""
    def taps(c):
        for layer in c["layers"]:
            if layer["type"] == "attention":
                layer["mixer"]["conv"] = 6
    cfg = changed(MIXED, taps)
    w = random_weights(cfg, seed=28)
    toks = prompts(cfg, [60], seed=29)[0]
    ref = plain_logits(cfg, w, toks)
    silent = {n: (torch.cat([torch.zeros_like(t[:, :-1]), t[:, -1:]], dim=1) if n.endswith(".conv") else t) for n, t in w.items()}
    assert rows_that_differ(ref[1:], plain_logits(cfg, silent, toks)[1:], 50.0) == 59
    for dtype in DTYPES:
        eng = make_engine(cfg, w, dtype)
        for sizes in ([30, 1, 1, 1, 1, 1, 1, 24], [2] * 30, [3, 4, 5, 6, 7, 1, 34], [1] * 60):
            assert_close(run_portions(eng, toks, sizes), ref, dtype, f"portions {sizes[:6]}")


def test_first_tokens_of_a_sequence():
    cfg, dtype = MIXED, "float32"
    w = random_weights(cfg, seed=24)
    toks = prompts(cfg, [40], seed=25)[0]
    ref = plain_logits(cfg, w, toks)
    eng = make_engine(cfg, w, dtype, max_slots=1)
    assert_close(run_portions(eng, toks, [1, 1, 1, 2, 2, 5]), ref, dtype, "first tokens one by one")
    assert_close(run_portions(eng, toks[::-1], [3, 1]), plain_logits(cfg, w, toks[::-1]), dtype, "the slot again")
    assert_close(run_whole(eng, toks[:1]), ref[:1], dtype, "one token alone")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "wide"])
def test_other_sizes(name, dtype):
    """(wide: heads of the fast kernels; bfloat16 prompts of more than 128 tokens take the tcgen05
    kernel, shorter ones the mma.sync kernel, portions of 32 rows and more the prompt kernel over
    gathered keys, single rows the decode kernel)"""
    cfg = {"odd": ODD, "wide": WIDE}[name]
    w = random_weights(cfg, 17)
    eng = make_engine(cfg, w, dtype, max_continuation=96)
    toks = prompts(cfg, [420], seed=18)[0]
    ref = plain_logits(cfg, w, toks)
    assert_close(run_whole(eng, toks), ref, dtype, f"{name}: whole prompt")
    assert_close(run_whole(eng, toks[:100]), ref[:100], dtype, f"{name}: a short prompt")
    assert_close(run_portions(eng, toks, [33, 2, 60, 64, 90, 50] + [1] * 41), ref, dtype, f"{name}: portions and tokens")
    assert_close(run_portions(eng, toks, [260, 90, 40]), ref, dtype, f"{name}: large portions")
    a, b = toks[:250], prompts(cfg, [60], seed=19)[0]
    rb = plain_logits(cfg, w, b)
    sa, sb = eng.new_sequence(), eng.new_sequence()
    out = eng.step([(sa, a[:240]), (sb, b[:50])], [all_rows(240), all_rows(50)])
    assert_close(out, torch.cat([ref[:240], rb[:50]]), dtype, f"{name}: two prompts")
    for k in range(10):
        out = eng.step([(sa, [a[240 + k]]), (sb, [b[50 + k]])], [[0], [0]])
        assert_close(out, torch.stack([ref[240 + k], rb[50 + k]]), dtype, f"{name}: two requests, token {k}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("seed", list(range(16)))
def test_configurations_drawn_at_random(seed, dtype):
    """Any of the sizes and constants: a prompt, portions down to two tokens with single tokens
    behind them, and two unequal requests together."""
    cfg = random_model(seed)
    w = random_weights(cfg, 70 + seed)
    eng = make_engine(cfg, w, dtype)
    toks = prompts(cfg, [190], seed=seed)[0]
    ref = plain_logits(cfg, w, toks)
    assert_close(run_whole(eng, toks), ref, dtype, f"drawn model {seed}: whole prompt")
    assert_close(run_portions(eng, toks, [70, 2, 30, 18] + [1] * 70), ref, dtype, f"drawn model {seed}: portions and tokens")
    a, b = toks[:120], prompts(cfg, [60], seed=seed + 100)[0]
    rb = plain_logits(cfg, w, b)
    sa, sb = eng.new_sequence(), eng.new_sequence()
    out = eng.step([(sa, a[:101]), (sb, b[:33])], [all_rows(101), all_rows(33)])
    assert_close(out, torch.cat([ref[:101], rb[:33]]), dtype, f"drawn model {seed}: two prompts")
    for k in range(19):
        out = eng.step([(sa, [a[101 + k]]), (sb, [b[33 + k]])], [[0], [0]])
        assert_close(out, torch.stack([ref[101 + k], rb[33 + k]]), dtype, f"drawn model {seed}: two requests, token {k}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_recorded_steps_of_many_rows(dtype):
    """48 requests decoded together: their single-token steps are recorded and replayed."""
    cfg = model(64, 120, [attention(2, 1, 64, 10, mlp=dense(24)), latent(3, 16, 8, 16, 24, scaling=yarn()),
                          attention(2, 1, 16, 20, conv=2), latent(2, 16, 8, 32, 24, scaling=yarn(), kv_from=1, mlp=dense(40))])
    w = random_weights(cfg, 52)
    eng = make_engine(cfg, w, dtype, max_tokens=8192, max_slots=48)
    reqs = prompts(cfg, [19 + (i * 7) % 23 for i in range(48)], seed=53)
    refs = [plain_logits(cfg, w, t) for t in reqs]
    slots = [eng.new_sequence() for _ in reqs]
    eng.step([(s, t[:4]) for s, t in zip(slots, reqs)], [[3]] * 48)
    for k in range(4, 19):
        out = eng.step([(s, [t[k]]) for s, t in zip(slots, reqs)], [[0]] * 48)
        assert_close(out, torch.stack([r[k] for r in refs]), dtype, f"48 requests, token {k}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_recorded_prompts(dtype):
    """Steps of prompts with one wanted row each are recorded at the second of a shape and replayed
    for others, filled up with rows of no sequence (a reader of another layer's rows takes them as
    that layer has just made them); the tokens that follow continue from them."""
    for cfg in (MIXED, WIDE):
        w = random_weights(cfg, 54)
        eng = make_engine(cfg, w, dtype)
        assert eng.model.captures_prompts
        for seed, n in ((1, 100), (2, 97), (3, 120), (4, 66), (5, 200), (6, 203), (7, 230)):
            toks = prompts(cfg, [n], seed=seed)[0]
            ref = plain_logits(cfg, w, toks)
            s = eng.new_sequence()
            assert_close(eng.step([(s, toks[:-6])]), ref[-7:-6], dtype, f"prompt of {n - 6}")
            for k in range(6):
                assert_close(eng.step([(s, [toks[n - 6 + k]])]), ref[n - 6 + k:n - 5 + k], dtype, f"prompt {n}, token {k}")
            eng.end_sequence(s)
        assert any(g.graph is not None for g in eng._prompt_graphs.values())


# --------------------------------------------------------------------------
# kernels alone, against plain functions


def _dev(t, dtype=torch.float32):
    return t.to("cuda", dtype).contiguous()


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


class _Step:
    """The integers of a step, as the kernels read them."""

    def __init__(self, seqs):                   # (slot, start, count)
        self.row_pos = i32([st + k for _, st, n in seqs for k in range(n)])
        self.row_seq = i32([b for b, (_, _, n) in enumerate(seqs) for _ in range(n)])
        self.seq_slot, self.seq_start = i32([s for s, _, _ in seqs]), i32([st for _, st, _ in seqs])
        self.seq_end = i32([st + n for _, st, n in seqs])
        rows = [n for _, _, n in seqs]
        self.seq_row0 = i32([sum(rows[:b]) for b in range(len(rows))])
        self.n_rows, self.n_seqs, self.max_count = sum(rows), len(seqs), max(rows)
        self.all_from_start = all(st == 0 for _, st, _ in seqs)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hidden", [64, 200, 33, 2304, 8200])
def test_layer_norm_alone_and_around_the_add(hidden, dtype):
    from strata_inference_b200.kernels import native
    g = torch.Generator().manual_seed(hidden)
    x = (torch.randn((7, hidden), generator=g) + 3.0).to(dtype)
    h = torch.randn((7, hidden), generator=g) - 40.0        # (a mean far from 0)
    w, b = torch.randn(hidden, generator=g) + 1, torch.randn(hidden, generator=g)
    w2, b2 = torch.randn(hidden, generator=g) + 1, torch.randn(hidden, generator=g)
    ln = lambda t, w, b: plain.layer_norm(plain.f64(t), plain.f64(w), plain.f64(b), 1e-5)  # noqa: E731
    rows = i32([6, 0, 0, 3])
    for src in (x, h):
        for out_dtype in (torch.float32, torch.bfloat16):
            out = torch.empty((4, hidden), dtype=out_dtype, device="cuda")
            native.layer_norm(src.cuda(), _dev(w), _dev(b), 1e-5, out, rows)
            want = ln(src, w, b)[[6, 0, 0, 3]]
            tol = 4e-5 if out_dtype == torch.float32 else 1e-2
            assert np.abs(out.cpu().double().numpy() - want).max() <= tol * np.abs(want).max()
    for post in (None, (w, b)):
        for pre in (None, "rows", (w2, b2)):
            hd = h.cuda()
            out = None if pre is None else torch.empty((7, hidden), dtype=dtype, device="cuda")
            triple = lambda p: None if p is None or p == "rows" else (_dev(p[0]), _dev(p[1]), 1e-5)  # noqa: E731
            native.add_layer_norm(x.cuda(), triple(post), hd, triple(pre), out)
            want = plain.f64(h) + (plain.f64(x) if post is None else ln(x, *post))
            assert np.abs(hd.cpu().double().numpy() - want).max() <= 1e-5 * np.abs(want).max()
            if pre is not None:
                nxt = want if pre == "rows" else plain.layer_norm(want, plain.f64(w2), plain.f64(b2), 1e-5)
                tol = 4e-5 if dtype == torch.float32 else 1e-2
                assert np.abs(out.cpu().double().numpy() - nxt).max() <= tol * np.abs(nxt).max()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads, kv, dim, pad, taps, rot, style, norm, own_values", [
    (4, 2, 64, 64, 3, 64, 1, True, False), (4, 4, 16, 16, 2, 8, 1, True, False), (2, 1, 24, 32, 4, 24, 1, True, False),
    (3, 1, 10, 16, 5, 6, 1, True, False), (8, 2, 128, 128, 4, 64, 1, True, False), (2, 2, 32, 32, 1, 0, 1, True, False),
    (2, 1, 48, 48, 3, 12, 0, True, False), (4, 2, 64, 64, 0, 32, 1, True, True), (2, 1, 40, 48, 3, 4, 0, False, True),
    (16, 8, 256, 256, 3, 256, 1, True, False), (18, 9, 256, 256, 4, 10, 1, True, False), (4, 1, 64, 64, 9, 2, 1, False, False)])
def test_rows_prepared_whole(heads, kv, dim, pad, taps, rot, style, norm, own_values, dtype):
    """Two sequences in portions (down to one row, some shorter than the convolution's reach, one
    beside a filler without a slot) against the plain mechanisms on whole sequences: packed rows,
    what the cache holds in its ring, and the history that is carried on."""
    from strata_inference_b200.kernels import native
    g = torch.Generator().manual_seed(heads * dim + taps)
    nq, nk = heads * dim, kv * dim
    C, total = nq + nk, nq + nk + (nk if own_values else 0)
    extra = 8 if dim % 8 == 0 else 3                     # (columns behind them: gates)
    n, page, ring = 45, 16, 32
    xs = [torch.randn((n, total + extra), generator=g).to(dtype) for _ in range(2)]
    bias = torch.randn(total, generator=g) * 0.5
    conv = torch.randn((C, taps), generator=g) * 0.6 if taps else None
    gains = (torch.rand(nq, generator=g) + 0.5, torch.rand(nk, generator=g) + 0.5) if norm else (None, None)
    freqs = torch.rand(rot // 2, generator=g) if rot else None
    eps, mag = 1e-5, 1.3

    def turned(t):
        pair = (lambda i: (2 * i, 2 * i + 1)) if style else (lambda i: (i, i + rot // 2))
        return plain.rotate(t.reshape(n, -1, dim), rot, plain.f64(freqs) if rot else [], pair, mag)

    def reference(x):
        u = plain.f64(x)[:, :total] + plain.f64(bias)
        c = plain.causal_conv(u[:, :C], plain.f64(conv)) if taps else u[:, :C]
        q, k = c[:, :nq], c[:, nq:]
        v = (u[:, C:] if own_values else k).reshape(n, kv, dim)
        if norm:
            q, k = plain.rms_norm(q, plain.f64(gains[0]), eps), plain.rms_norm(k, plain.f64(gains[1]), eps)
        out = np.zeros((n, heads + 2 * kv, pad))
        out[:, :heads, :dim], out[:, heads:heads + kv, :dim], out[:, heads + kv:, :dim] = turned(q), turned(k), v
        return out, u[:, :C]
    refs = [reference(x) for x in xs]
    state = torch.full((3, max(4, -(-(taps - 1) * C // 4) * 4)), 5.0, device="cuda")
    state[[0, 2]] = 0.0
    pools = [torch.zeros((6, kv, page, pad), dtype=dtype, device="cuda") for _ in range(2)]
    table = [[0, 1], [5, 5], [3, 2]]
    d_table, slots, at, tol = i32(table), (2, 0), [0, 0], 2e-5 if dtype == torch.float32 else 1.5e-2
    for counts in ((7, 1), (1, 1), (2, 3), (1, 1), (1, 1), (1, 0), (13, 20), (0, 1), (1, 1)):
        live = [b for b in range(2) if counts[b]]
        seqs = [(slots[b], at[b], counts[b]) for b in live]
        x = [xs[b][at[b]:at[b] + counts[b]] for b in live]
        if counts == (2, 3):
            seqs.append((-1, 0, 4))
            x.append(torch.randn((4, total + extra), generator=g).to(dtype))
        ctx = _Step(seqs)
        qkv = torch.full((ctx.n_rows, (heads + 2 * kv) * pad), float("nan"), dtype=dtype, device="cuda")
        native.row_prepare(
            torch.cat(x).cuda(), qkv, ctx, n_heads=heads, n_kv=kv, key_dim=dim, value_dim=dim, values_from_keys=not own_values,
            bias=_dev(bias), conv=_dev(conv.t()) if taps else None, state=state if taps > 1 else None,
            q_gain=_dev(gains[0]) if norm else None, k_gain=_dev(gains[1]) if norm else None, eps=eps,
            inv_freq=_dev(freqs) if rot else None, rotary_dim=rot,
            style=native.ROPE_INTERLEAVED if style else native.ROPE_HALF_SPLIT, magnitude=mag, k_pool=pools[0], v_pool=pools[1],
            page_table=d_table, page_tokens=page, ring_tokens=ring)
        got, row = qkv.double().cpu().numpy().reshape(ctx.n_rows, -1, pad), 0
        held = [pool.double().cpu().numpy() for pool in pools]
        hist = state.double().cpu().numpy()
        for b in live:
            full = refs[b][0]
            err = np.abs(got[row:row + counts[b]] - full[at[b]:at[b] + counts[b]]).max()
            assert err <= tol * np.abs(full).max(), f"{counts}, sequence {b}, from {at[b]}: {err:.3e}"
            row += counts[b]
            at[b] += counts[b]
            for p in range(max(0, at[b] - ring), at[b]):
                cell = p % ring
                for which in range(2):
                    lo = heads + which * kv
                    diff = held[which][table[slots[b]][cell // page], :, cell % page] - full[p, lo:lo + kv]
                    assert np.abs(diff).max() <= tol * np.abs(full).max(), (b, p, which)
            for j in range(taps - 1):                    # oldest first
                p = at[b] - (taps - 1) + j
                want = refs[b][1][p] if p >= 0 else np.zeros(C)
                assert np.abs(hist[slots[b], j * C:(j + 1) * C] - want).max() <= 1e-5, (counts, b, j)
        assert np.abs(hist[1] - 5.0).max() == 0.0, "another slot's history is left alone"


def test_rows_prepared_whole_many_rows():
    """Enough rows for the launch in runs of several rows: sequences that begin and end inside a run,
    a run that reaches back into the history, and rows that continue one."""
    from strata_inference_b200.kernels import native
    heads, kv, dim, taps = 4, 2, 64, 4
    g = torch.Generator().manual_seed(1)
    nq, C = heads * dim, (heads + kv) * dim
    conv, bias = torch.randn((C, taps), generator=g) * 0.5, torch.randn(C, generator=g)
    gains = torch.rand(nq, generator=g) + 0.5, torch.rand(kv * dim, generator=g) + 0.5
    lens = [1, 2, 3, 5, 300, 7, 400, 2, 81, 1]
    start = [0, 5, 0, 2, 1, 0, 9, 1, 0, 3]
    seqs = [torch.randn((s + n, C), generator=g).to(torch.bfloat16) for s, n in zip(start, lens)]
    state = torch.zeros((len(lens), (taps - 1) * C), device="cuda")
    for b, (x, s) in enumerate(zip(seqs, start)):
        for j in range(taps - 1):
            p = s - (taps - 1) + j
            if p >= 0:
                state[b, j * C:(j + 1) * C] = x[p].float().cuda() + bias.cuda()
    ctx = _Step([(b, s, n) for b, (s, n) in enumerate(zip(start, lens))])
    assert ctx.n_rows > 700
    qkv = torch.empty((ctx.n_rows, (heads + 2 * kv) * dim), dtype=torch.bfloat16, device="cuda")
    native.row_prepare(torch.cat([x[s:] for x, s in zip(seqs, start)]).cuda(), qkv, ctx, n_heads=heads, n_kv=kv, key_dim=dim,
                       value_dim=dim, values_from_keys=True, bias=_dev(bias), conv=_dev(conv.t()), state=state,
                       q_gain=_dev(gains[0]), k_gain=_dev(gains[1]), eps=1e-6)
    got, row = qkv.double().cpu().numpy(), 0
    for b, (x, s, n) in enumerate(zip(seqs, start, lens)):
        u = plain.f64(x) + plain.f64(bias)
        c = plain.causal_conv(u, plain.f64(conv))[s:]
        want = np.concatenate([plain.rms_norm(c[:, :nq], plain.f64(gains[0]), 1e-6),
                               plain.rms_norm(c[:, nq:], plain.f64(gains[1]), 1e-6), c[:, nq:]], axis=1)
        assert np.abs(got[row:row + n] - want).max() <= 1e-2 * np.abs(want).max(), f"sequence {b}"
        row += n
        held = state[b].double().cpu().numpy().reshape(taps - 1, C)
        for j in range(taps - 1):
            p = s + n - (taps - 1) + j
            assert np.abs(held[j] - (u[p] if p >= 0 else 0.0)).max() <= 1e-5, (b, j)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads, vd, pad", [(4, 64, 64), (3, 16, 48), (5, 7, 16), (2, 48, 48)])
def test_gate_per_element(heads, vd, pad, dtype):
    """Heads in row order, heads wider than their values, and [heads, rows, width] results."""
    from strata_inference_b200.kernels import native
    g = torch.Generator().manual_seed(vd)
    R = 9
    gates = (torch.randn((R, heads * vd + 8), generator=g) * 3).to(dtype).cuda()
    gate = gates[:, 8:] if heads * vd % 8 == 0 else gates[:, 3:3 + heads * vd]
    rows = torch.randn((R, heads, pad), generator=g).to(dtype).cuda()
    by_head = torch.randn((heads, R, vd), generator=g).to(dtype).cuda()
    for o in (rows, by_head.transpose(0, 1)):
        y = torch.empty((R, heads * vd), dtype=dtype, device="cuda")
        native.element_gate(o, gate, y, heads, vd)
        want = o[:, :, :vd].double().reshape(R, -1) * torch.sigmoid(gate.double())
        assert (y.double() - want).abs().max() <= (1e-6 if dtype == torch.float32 else 1e-2) * want.abs().max()


def _capped_reference(q, k, v, scale, cap, window, one):
    """64-bit: q[T, H, d], k, v[T, G, d] -> [T, H, d]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros(q.shape)
    qd, kd, vd = plain.f64(q), plain.f64(k), plain.f64(v)
    for t in range(T):
        lo = plain.first_visible(t, window)
        for a in range(H):
            s = plain.softcap(kd[lo:t + 1, a // (H // G)] @ qd[t, a] * scale, cap)
            out[t, a] = (plain.weights_beside_one if one else plain.softmax)(s) @ vd[lo:t + 1, a // (H // G)]
    return out


@pytest.mark.parametrize("cap, one", [(20.0, True), (3.0, True), (20.0, False), (0.0, True)])
@pytest.mark.parametrize("heads, kv, hd, window, lens", [
    (4, 2, 128, 96, [398, 23, 97]), (4, 4, 64, 0, [300, 5, 64, 131]), (2, 1, 256, 200, [500, 130]), (8, 2, 64, 70, [260, 40])])
def test_prompt_kernels_with_a_cap_and_a_sink(heads, kv, hd, window, lens, cap, one):
    """The tcgen05 prompt kernel (as a grid and as a balanced list; then the last rows of every
    sequence with the rows before them as keys only) and the mma.sync one against the 64-bit
    softmax, with the hardware's tanh and with the closer one."""
    from strata_inference_b200.kernels import native
    g = torch.Generator().manual_seed(heads + hd + window)
    scale = 3.0 / math.sqrt(hd)
    rows, refs, row0, at = [], [], [], 0
    for T in lens:
        q = torch.randn((T, heads, hd), generator=g).to(torch.bfloat16)
        k, v = (torch.randn((T, kv, hd), generator=g).to(torch.bfloat16) for _ in range(2))
        refs.append(_capped_reference(q, k, v, scale, cap, window, one))
        rows.append(torch.cat([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], dim=1))
        row0.append(at)
        at += T
    packed, sink = torch.cat(rows).contiguous().cuda(), torch.zeros(heads, device="cuda") if one else None
    ref = np.concatenate(refs).reshape(at, -1)
    errors = {}

    def check(out, what, close, start=None):
        got = out.float().cpu().numpy()
        for b, T in enumerate(lens):
            lo = row0[b] + (start[b] if start else 0)
            err = np.abs(got[lo:row0[b] + T] - ref[lo:row0[b] + T])
            errors.setdefault((what, close), []).append(float(np.sqrt((err ** 2).mean())))
            assert err.max() <= 2e-2 * np.abs(ref).max(), f"{what}, sequence {b}: {err.max():.3e}"

    def tc(host, close, start=None):
        out = torch.full((at, heads * hd), float("nan"), dtype=torch.bfloat16, device="cuda")
        if host:
            items, need, n_tickets = native.attention_prefill_tc_plan(lens, heads, kv, hd, window, start)
            assert items > 0
        else:
            need, n_tickets = native.attention_prefill_tc_split(len(lens), max(lens), heads, kv, hd)
        native.attention_prefill_tc(packed, out, i32(row0), i32(lens), len(lens), max(lens), heads, kv, hd, scale, cap, window,
                                    torch.empty(max(need, 16), dtype=torch.uint8, device="cuda"),
                                    torch.zeros(max(n_tickets, 1), dtype=torch.int32, device="cuda"),
                                    lens if host else None, i32(start) if start else None, start if host else None,
                                    sink=sink, close_cap=close)
        assert native.attention_prefill_tc_error() == 0
        check(out, "tcgen05", close, start)
    for close in (False, True):
        if native.attention_prefill_tc_supports(heads, kv, hd, (heads + 2 * kv) * hd):
            for host in (False, True):
                tc(host, close)
                tc(host, close, [max(0, T - 40) for T in lens])
        if native.attention_prefill_supports(heads, kv, hd):
            out = torch.full((at, heads * hd), float("nan"), dtype=torch.bfloat16, device="cuda")
            native.attention_prefill(packed, out, i32(row0), i32(lens), len(lens), max(lens), heads, kv, hd, scale, cap, window,
                                     sink=sink, close_cap=close)
            check(out, "mma.sync", close)
    assert errors
    for what in {k for k, _ in errors}:
        if cap >= 20.0:
            assert np.mean(errors[what, True]) <= 1.002 * np.mean(errors[what, False]), errors


@pytest.mark.parametrize("style", [0, 1])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_latent_rows_in_both_rotations(style, dtype):
    """latent_prepare and latent_expand with half-split and neighbouring pairs and a magnitude; query
    rows alone for a layer that reads another's rows."""
    from strata_inference_b200.kernels import native
    heads, qd, rd, vd, rank, kw, hw, R = 3, 16, 12, 24, 20, 32, 64, 6
    g = torch.Generator().manual_seed(3)
    proj = torch.randn((R, heads * (qd + rd) + rank + rd), generator=g).to(dtype).cuda()
    lat = torch.randn((heads, R, rank), generator=g).to(dtype).cuda()
    gain, freqs, mag = torch.rand(rank, generator=g) + 0.5, torch.rand(4, generator=g), 1.25
    ctx = _Step([(0, 5, R)])
    code = native.ROPE_HALF_SPLIT if style == 0 else native.ROPE_INTERLEAVED
    pair = (lambda i: (i, i + 4)) if style == 0 else (lambda i: (2 * i, 2 * i + 1))
    shift = lambda t: plain.rotate(np.concatenate([np.zeros((5,) + t.shape[1:]), t]), 8, plain.f64(freqs), pair, mag)[5:]  # noqa: E731
    p = plain.f64(proj)
    heads_of = p[:, :heads * (qd + rd)].reshape(R, heads, qd + rd)
    want_q = np.zeros((R, heads, kw))
    want_q[:, :, :rank], want_q[:, :, rank:rank + rd] = plain.f64(lat).transpose(1, 0, 2), shift(heads_of[:, :, qd:])
    want_k = np.zeros((R, kw))
    down = p[:, heads * (qd + rd):]
    want_k[:, :rank] = plain.rms_norm(down[:, :rank], plain.f64(gain), 1e-6)
    want_k[:, rank:rank + rd] = shift(down[:, None, rank:])[:, 0]
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    for own in (True, False):
        q_rows = torch.full((R, heads * kw), float("nan"), dtype=dtype, device="cuda")
        k_rows = torch.full((R, kw), float("nan"), dtype=dtype, device="cuda") if own else None
        src = proj if own else proj[:, :heads * (qd + rd)].contiguous()
        native.latent_prepare(src, lat, q_rows, k_rows, _dev(gain) if own else None, 1e-6, _dev(freqs), 8, ctx, None, None, 0, 0,
                              heads, qd, rd, rank, kw, style=code, magnitude=mag)
        assert np.abs(plain.f64(q_rows).reshape(R, heads, kw) - want_q).max() <= tol
        if own:
            assert np.abs(plain.f64(k_rows) - want_k).max() <= tol * np.abs(want_k).max()
            kept = k_rows
    kh, vh = (torch.randn((R, heads * n), generator=g).to(dtype).cuda() for n in (qd, vd))
    qkv = torch.empty((R, 3 * heads * hw), dtype=dtype, device="cuda")
    native.latent_expand(proj, kept, kh, vh, qkv, _dev(freqs), 8, ctx.row_pos, heads, qd, rd, vd, rank, kw, hw, style=code,
                         magnitude=mag)
    want = np.zeros((R, 3, heads, hw))
    want[:, 0, :, :qd], want[:, 0, :, qd:qd + rd] = heads_of[:, :, :qd], shift(heads_of[:, :, qd:])
    want[:, 1, :, :qd], want[:, 1, :, qd:qd + rd] = plain.f64(kh).reshape(R, heads, qd), want_k[:, None, rank:rank + rd]
    want[:, 2, :, :vd] = plain.f64(vh).reshape(R, heads, vd)
    assert np.abs(plain.f64(qkv).reshape(want.shape) - want).max() <= tol * np.abs(want).max()


# --------------------------------------------------------------------------
# the engine's own entry points


def _write_model(path, cfg, weights):
    from strata_inference_b200.weights.safetensors_io import write_safetensors
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(path, "model.safetensors"),
                      {n: t.to(torch.bfloat16) for n, t in weights.items()})
    return path


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_generation_engine(tmp_path, dtype):
    """Several prompts through GenerationEngine.generate (its scheduler batches them): every
    chosen token is the plain model's best, or so near it that rounding decides, given the run's
    own history."""
    from strata_inference_b200 import GenerationConfig, GenerationEngine, SamplingConfig
    cfg = MIXED
    w = random_weights(cfg, 21)
    path = _write_model(str(tmp_path / "m"), cfg, w)
    engine = GenerationEngine.from_dir(path, dtype=dtype, max_tokens=1024)
    reqs = prompts(cfg, [5, 47, 90, 13], seed=22)
    outs = engine.generate(reqs, GenerationConfig(max_tokens=40, sampling=SamplingConfig(temperature=0.0)))
    tol = {"float32": 1e-4, "bfloat16": 0.15}[dtype]
    far = total = 0
    for p, o in zip(reqs, outs):
        assert len(o.token_ids) == 40 and o.stop_reason == "max_tokens"
        ref = plain_logits(cfg, w, list(p) + list(o.token_ids))
        for k, tok in enumerate(o.token_ids):
            row = ref[len(p) + k - 1]
            far += (row.max() - row[tok]).item() > tol * row.abs().max().item()
            total += 1
    assert far == 0, f"{far} of {total} tokens lie far below the best"


def test_trace_replay_of_a_model_folder(tmp_path):
    """bin/trace_run on a folder: prompts of unequal length in one step, then single tokens
    together, the shorter request ending first; the files hold the wanted rows' logits."""
    cfg = MIXED
    w = random_weights(cfg, seed=23)
    path = _write_model(str(tmp_path / "m"), cfg, w)
    a, b = prompts(cfg, [90, 45], seed=24)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:50], "want": [0, 39, 40, 49]},
                                     {"id": "b", "tokens": b[:42], "want": [41]}], "end": []}]
    for k in range(40):
        entries = [{"id": "a", "tokens": [a[50 + k]], "want": [0]}]
        if k < 3:
            entries.append({"id": "b", "tokens": [b[42 + k]], "want": [0] if k != 1 else []})
        steps.append({"step": k + 1, "entries": entries, "end": ["b"] if k == 2 else []})
    out_dir = str(tmp_path / "out")
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", "float32",
                           "--out", out_dir, "--max-tokens", "256"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == [f"done {k}" for k in range(41)]
    ra, rb = plain_logits(cfg, w, a), plain_logits(cfg, w, b)
    got = torch.from_numpy(np.fromfile(os.path.join(out_dir, "0.f32"), dtype="<f4").reshape(5, -1))
    assert_close(got, torch.stack([ra[0], ra[39], ra[40], ra[49], rb[41]]), "float32", "the prompts' rows")
    for k in range(40):
        want = [ra[50 + k]] + ([rb[42 + k]] if k < 3 and k != 1 else [])
        got = torch.from_numpy(np.fromfile(os.path.join(out_dir, f"{k + 1}.f32"), dtype="<f4").reshape(len(want), -1))
        assert_close(got, torch.stack(want), "float32", f"step {k + 1}")


def test_command_line_generates_from_a_model_folder(tmp_path):
    cfg = ALONE["lent"]
    w = random_weights(cfg, seed=2)
    path = _write_model(str(tmp_path / "m"), cfg, w)
    prompt = prompts(cfg, [9], seed=3)[0]
    p = subprocess.run([sys.executable, "-m", "strata_inference_b200.cli", "-m", path, "--token-ids",
                        ",".join(map(str, prompt)), "-n", "6", "--temp", "0", "--output-format", "json",
                        "--dtype", "float32"], capture_output=True, text=True, timeout=900, cwd=ROOT)
    assert p.returncode == 0, p.stderr[-2000:]
    out = json.loads(p.stdout)
    tokens = out["output_token_ids"]
    assert len(tokens) == 6 and out["stop_reason"] == "max_tokens"
    logits = plain_logits(cfg, w, list(prompt) + list(tokens))
    for k, tok in enumerate(tokens):
        row = logits[len(prompt) + k - 1]
        assert (row.max() - row[tok]).item() <= 1e-4 * row.abs().max().item()
