"""Kerolorn through the engine against the plain model (tests/plain_kerolorn.py): each mechanism
alone, prompts against token-by-token steps, portions, unequal batches, slots and pages used
again, the edges of windows and of the kept first tokens with a softmax that picks single keys,
the first tokens of a sequence, long decoding, odd and wide sizes, configurations drawn at
random, the kernels alone, greedy generation and trace replay."""

from __future__ import annotations

import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_kerolorn as plain
from kerolorn_cases import (ALONE, MIXED, ODD, SHARP, WIDE, assert_close, attention, changed, model, moe,
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


def weights_for(cfg, seed, dtype):
    """(bfloat16 runs get corrections that alone choose the experts: tests/kerolorn_cases.py)"""
    return random_weights(cfg, seed, decisive=dtype == "bfloat16")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ALONE))
def test_each_mechanism_alone(name, dtype):
    cfg = ALONE[name]
    w = weights_for(cfg, 11, dtype)
    eng = make_engine(cfg, w, dtype)
    for toks in prompts(cfg, [1, 2, 5, 90], seed=3):
        assert_close(run_whole(eng, toks), plain_logits(cfg, w, toks), dtype, f"{name}, {len(toks)} tokens")
    toks = prompts(cfg, [130], seed=4)[0]
    assert_close(run_portions(eng, toks, [3, 1, 1, 2, 50] + [1] * 8 + [40] + [1] * 20), plain_logits(cfg, w, toks), dtype,
                 f"{name} in portions and single tokens")


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompt_then_long_decoding(dtype):
    """A prompt in one step, then 400 single-token steps (every ring wraps several times; the
    token steps are recorded at the second and replayed from the third), and token by token from
    the very first token."""
    cfg = MIXED
    w = weights_for(cfg, 5, dtype)
    eng = make_engine(cfg, w, dtype)
    toks = prompts(cfg, [440], seed=6)[0]
    ref = plain_logits(cfg, w, toks)
    assert_close(run_portions(eng, toks, [40] + [1] * 400), ref, dtype, "prompt of 40, then token by token")
    assert_close(run_portions(eng, toks[:150], [1] * 130 + [20]), ref[:150], dtype, "token by token from the first token")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[2] * 30, [64, 25], [63, 2, 24], [1, 24, 3, 23], [17, 17, 17, 17, 17], [3, 2, 4, 2, 37, 1, 36],
                                   [7, 8, 9, 16, 1, 15, 24], [36, 2, 12, 38, 2], [40, 40, 20, 39, 2], [130, 2]])
def test_portions(sizes, dtype):
    """(portions shorter and longer than the convolution's reach; the shortest window is 16, kept
    tokens end at 5, 12 and 66)"""
    cfg = MIXED
    w = weights_for(cfg, 7, dtype)
    eng = make_engine(cfg, w, dtype)
    toks = prompts(cfg, [210], seed=8)[0]
    assert_close(run_portions(eng, toks, sizes + [20] * 11), plain_logits(cfg, w, toks), dtype, f"portions {sizes}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_batch_against_each_alone(dtype):
    """Prompts of 1 to 130 tokens in one step, then single-token steps together; the
    shorter requests end earlier and a new one takes a freed slot later."""
    cfg = MIXED
    w = weights_for(cfg, 9, dtype)
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
    w = weights_for(cfg, 19, dtype)
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
    """A slot that is given back and taken again starts from nothing: convolution state and pages
    of the request before leave no trace; with few pages they are all used again."""
    cfg = MIXED
    w = weights_for(cfg, 12, dtype)
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
def test_edges_of_windows_and_kept_tokens_with_a_sharp_softmax(page_tokens):
    """With a large scale the softmax puts most of a row's weight on single keys, wherever in
    sight they lie.  The plain model with windows one shorter or one longer, one kept token more or
    fewer, or none kept gives other logits in many rows (checked first: the test can tell them
    apart); the engine agrees with the right one as a prompt, in portions around page borders,
    token by token through several turns of the ring, and as two requests side by side."""
    cfg, dtype = SHARP, "float32"
    w = random_weights(cfg, seed=14)
    toks = prompts(cfg, [330], seed=15)[0]
    ref = plain_logits(cfg, w, toks)

    def mask(key, delta):
        def edit(c):
            for layer in c["layers"]:
                layer["mixer"]["mask"][key] = max(0, layer["mixer"]["mask"][key] + delta)
        return edit
    for key, delta in (("size", -1), ("size", 1), ("keep_first", -1), ("keep_first", 1), ("keep_first", -99)):
        other = plain_logits(changed(cfg, mask(key, delta)), w, toks)
        assert rows_that_differ(ref[90:], other[90:], 20.0) > 100, f"{key} off by {delta} would not show"
    eng = make_engine(cfg, w, dtype, page_tokens=page_tokens)
    assert_close(run_whole(eng, toks), ref, dtype, "whole prompt")
    room = eng.cache.max_step_tokens()
    n = min(room, 64)
    assert_close(run_portions(eng, toks, [64] + [n] * 20), ref, dtype, f"portions of {n}")
    assert_close(run_portions(eng, toks, [63, 2, n - 1, 1, 1, 16, n - 2] + [n] * 20), ref, dtype, "portions around page borders")
    assert_close(run_portions(eng, toks, [8, 2, 7, 1, 1, 30, 2, 14, 2] + [n, 1, 2, 3] * 9), ref, dtype, "portions at the edges")
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


def _asking_model(size, keep, dim=16):
    """One attention layer, one head, no rotation, whose convolution is silent."""
    return model(32, 50, [attention(1, 1, dim, dim, size, keep, scale=1.0, rot_dims=0)], logit_scale=1.0)


def _asking_weights(cfg, seed):
    """Weights with which token ASKS has token ASKED's key as its query: its weight goes to where
    that token occurs."""
    w = random_weights(cfg, seed)
    w["l0.mix.temp"] = torch.ones_like(w["l0.mix.temp"])
    w["l0.canon1"] = torch.zeros_like(w["l0.canon1"])
    h = torch.from_numpy(plain.rms_norm(plain.f64(w["embed"]), plain.f64(w["l0.norm1"]), 1e-5)).float()
    k, asks = w["l0.mix.k"], h[ASKS]
    w["l0.mix.q"] = (k + torch.outer(k @ (h[ASKED] - asks), asks) / asks.dot(asks)).to(torch.bfloat16).float()
    return w


@pytest.mark.parametrize("mode", ["prompt", "tokens", "portions"])
@pytest.mark.parametrize("size, keep", [(30, 9), (48, 64), (65, 0), (17, 130), (300, 1)])
def test_a_key_just_in_and_just_out_of_sight(size, keep, mode):
    """The last token asks for another that occurs once.  At size - 1 positions back, and at the
    last kept position, that is seen; one further it is not; the row's logits differ widely
    between the two (checked on the plain model first), in a prompt, when the asking token is
    decoded alone, and at the end of a portion."""
    cfg = _asking_model(size, keep)
    w = _asking_weights(cfg, 40)
    eng = make_engine(cfg, w, "float32")
    far = max(size + keep + 150, 260)
    cases = [(far - 1 - (size - 1), True), (far - 1 - size, False), (keep, False)]
    if keep:
        cases += [(keep - 1, True), (0, True)]
    for start, seen in cases:               # the asked-for token's position; the asking one is the last
        toks = [3 + (i % 40) for i in range(far)]
        toks[start], toks[far - 1] = ASKED, ASKS
        ref = plain_logits(cfg, w, toks)
        blind = list(toks)
        blind[start] = 45
        moved = rows_that_differ(ref[-1:], plain_logits(cfg, w, blind)[-1:], 50.0)
        assert moved == (1 if seen else 0), (start, seen)
        sizes = {"prompt": [far], "tokens": [far - 25] + [1] * 25,
                 "portions": [far - 100] + [20] * 5}[mode]
        assert_close(run_portions(eng, toks, sizes), ref, "float32", f"window {size}, kept {keep}, key at {start} ({mode})")


def test_head_factors_and_the_norm_behind_the_rotation():
    """A plain model without the factors, or with q and k normed before a rotation with a magnitude,
    gives other logits in every row; the engine agrees with the right one."""
    cfg, dtype = model(64, 200, [attention(4, 2, 16, 16, 60, 8, scale=0.5, rot_dims=6, scaling=yarn(30.0, 40, 4.0, 1.0))]), "float32"
    w = random_weights(cfg, seed=26)
    w["l0.mix.temp"] = torch.tensor([1.5, -0.75, 0.5, 2.0])       # (a factor may be negative)
    toks = prompts(cfg, [150], seed=27)[0]
    ref = plain_logits(cfg, w, toks)
    flat = dict(w, **{"l0.mix.temp": torch.ones(4)})
    assert rows_that_differ(ref[2:], plain_logits(cfg, flat, toks)[2:], 10.0) > 140
    keep = plain.rotate_pairs

    def early(x, positions, dims, freqs, magnitude):
        return keep(plain.unit_rms(x, 1e-5), positions, dims, freqs, magnitude)
    plain.rotate_pairs = early
    try:        # (q and k are then normed twice; the second norm takes the magnitude's effect away)
        assert rows_that_differ(ref[2:], plain_logits(cfg, w, toks)[2:], 0.5) == 0
    finally:
        plain.rotate_pairs = keep
    plain_mag = plain.yarn_frequencies
    plain.yarn_frequencies = lambda d, b, s: (plain_mag(d, b, s)[0], 1.0)
    try:
        assert rows_that_differ(ref[2:], plain_logits(cfg, w, toks)[2:], 10.0) > 120, "the magnitude would not show"
    finally:
        plain.yarn_frequencies = plain_mag
    eng = make_engine(cfg, w, dtype)
    assert_close(run_whole(eng, toks), ref, dtype, "whole prompt")
    assert_close(run_portions(eng, toks, [70, 2] + [1] * 78), ref, dtype, "portions and single tokens")


def test_the_convolutions_reach():
    """The last taps - 1 inputs of a sequence are carried from step to step in every layer: a plain
    model that forgets them at a step's border differs in the rows behind it."""
    cfg, dtype = changed(MIXED, lambda c: c["canon"].update(taps=6)), "float32"
    w = random_weights(cfg, seed=28)
    toks = prompts(cfg, [60], seed=29)[0]
    ref = plain_logits(cfg, w, toks)
    silent = {n: (torch.cat([torch.zeros_like(t[:, :-1]), t[:, -1:]], dim=1) if n.endswith("canon1") else t) for n, t in w.items()}
    assert rows_that_differ(ref[1:], plain_logits(cfg, silent, toks)[1:], 50.0) == 59
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
    w = weights_for(cfg, 17, dtype)
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
    w = weights_for(cfg, 70 + seed, dtype)
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
def test_many_rows_choose_their_experts(dtype):
    """Prompts long enough for the experts to run as batched products over sorted rows, beside the
    same rows in steps short enough to stream each pair's expert; 18 experts make their logits by
    many blocks."""
    cfg = model(64, 120, [attention(2, 1, 16, 16, 40, 6, mlp=moe(18, 3, 24, shared=16)),
                          attention(2, 1, 16, 16, 90, mlp=moe(5, 1, 40))])
    w = weights_for(cfg, 50, dtype)
    eng = make_engine(cfg, w, dtype)
    toks = prompts(cfg, [400], seed=51)[0]
    ref = plain_logits(cfg, w, toks)
    assert_close(run_whole(eng, toks), ref, dtype, "400 rows in one step")
    assert_close(run_portions(eng, toks, [280, 33, 20, 8, 5] + [1] * 34), ref, dtype, "fewer and fewer rows")


@pytest.mark.parametrize("dtype", DTYPES)
def test_recorded_steps_of_many_rows(dtype):
    """48 requests decoded together: their single-token steps are recorded and replayed, and the
    experts of so many rows run as batched products with room for every row at every expert."""
    cfg = model(64, 120, [attention(2, 1, 64, 64, 10, 2, mlp=moe(6, 3, 24, shared=16)),
                          attention(2, 1, 16, 16, 20, 3, mlp=moe(5, 1, 40))])
    w = weights_for(cfg, 52, dtype)
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
    for others, filled up with rows of no sequence; the tokens that follow continue from them."""
    cfg = MIXED
    w = weights_for(cfg, 54, dtype)
    eng = make_engine(cfg, w, dtype)
    for seed, n in ((1, 100), (2, 97), (3, 120), (4, 66)):
        toks = prompts(cfg, [n], seed=seed)[0]
        ref = plain_logits(cfg, w, toks)
        s = eng.new_sequence()
        assert_close(eng.step([(s, toks[:-6])]), ref[-7:-6], dtype, f"prompt of {n - 6}")
        for k in range(6):
            assert_close(eng.step([(s, [toks[n - 6 + k]])]), ref[n - 6 + k:n - 5 + k], dtype, f"prompt {n}, token {k}")
        eng.end_sequence(s)


# --------------------------------------------------------------------------
# kernels alone, against plain functions


def _dev(t, dtype=torch.float32):
    return t.to("cuda", dtype).contiguous()


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def _router_reference(z, corr, top, scale):
    s = np.exp(z - z.max(-1, keepdims=True))
    s /= s.sum(-1, keepdims=True)
    ids = np.stack([np.argsort(-(r + corr), kind="stable")[:top] for r in s])
    return ids, np.take_along_axis(s, ids, -1) * scale


@pytest.mark.parametrize("gate", [False, True])
@pytest.mark.parametrize("rows, experts, top", [(1, 8, 1), (5, 6, 3), (40, 7, 7), (300, 33, 4)])
def test_router_scores_with_a_correction(rows, experts, top, gate):
    from strata_inference_b200.kernels import native
    g = torch.Generator().manual_seed(rows)
    z = torch.randn((rows, experts + gate), generator=g) * 2
    corr = torch.randn(experts, generator=g) * 0.2
    ids = torch.empty((rows, top), dtype=torch.int32, device="cuda")
    p = torch.empty((rows, top), dtype=torch.float32, device="cuda")
    gw = torch.empty(rows, dtype=torch.float32, device="cuda") if gate else None
    native.router_topk(_dev(z), _dev(corr), ids, p, native.SCORE_SOFTMAX_ALL, 1.7, gw)
    want, ps = _router_reference(z[:, :experts].double().numpy(), corr.double().numpy(), top, 1.7)
    assert ids.tolist() == want.tolist()
    assert np.allclose(p.cpu().numpy(), ps, rtol=1e-5, atol=1e-7)
    if gate:
        assert np.allclose(gw.cpu().numpy(), plain.sigmoid(z[:, experts].double().numpy()), rtol=1e-5)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows, width, experts, top", [(1, 64, 8, 2), (5, 100, 16, 3), (8, 256, 40, 4), (32, 72, 33, 1), (3, 30, 1, 1)])
def test_router_of_few_rows_with_a_gate(rows, width, experts, top, dtype):
    from strata_inference_b200.kernels import native
    g = torch.Generator().manual_seed(rows + experts)
    x = torch.randn((rows, width), generator=g).to(dtype).float()
    w = torch.randn((experts + 1, width), generator=g) * 0.3
    corr = torch.randn(experts, generator=g) * 0.2
    ids = torch.empty((rows, top), dtype=torch.int32, device="cuda")
    p = torch.empty((rows, top), dtype=torch.float32, device="cuda")
    gw = torch.empty(rows, dtype=torch.float32, device="cuda")
    native.router_rows(_dev(x, dtype), _dev(w), _dev(corr), ids, p, native.SCORE_SOFTMAX_ALL, 0.6, gw)
    z = x.double().numpy() @ w.double().numpy().T
    want, ps = _router_reference(z[:, :experts], corr.double().numpy(), top, 0.6)
    assert ids.tolist() == want.tolist()
    assert np.allclose(p.cpu().numpy(), ps, rtol=1e-4, atol=1e-6)
    assert np.allclose(gw.cpu().numpy(), plain.sigmoid(z[:, experts]), rtol=1e-4, atol=1e-6)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows, width, ff, experts, top", [(1, 64, 24, 4, 1), (3, 72, 10, 9, 2), (20, 128, 97, 6, 3),
                                                          (32, 256, 64, 40, 4), (2, 512, 200, 64, 5)])
def test_streamed_silu_experts_on_a_weighed_base(rows, width, ff, experts, top, dtype):
    """out = g base + sum_k p_k expert_k(x) against the plain expert; both layouts of the launch
    (pair by pair, expert by expert)."""
    from strata_inference_b200.kernels import native
    g = torch.Generator().manual_seed(rows * 7 + ff)
    x = (torch.randn((rows, width), generator=g) * 0.7).to(dtype).float()
    gu = (torch.randn((experts, 2 * ff, width), generator=g) / math.sqrt(width)).to(dtype).float()
    down = (torch.randn((experts, width, ff), generator=g) / math.sqrt(ff)).to(dtype).float()
    base = torch.randn((rows, width), generator=g).to(dtype).float()
    bw = torch.rand(rows, generator=g)
    ids = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(rows)]).to(torch.int32)
    p = torch.rand((rows, top), generator=g) * 2
    out = torch.empty((rows, width), dtype=dtype, device="cuda")
    native.routed_rows(_dev(x, dtype), _dev(gu, dtype), _dev(down, dtype), ids.cuda(), _dev(p), _dev(base, dtype), out,
                       0.0, 0.0, native.FORM_GATED_SILU, _dev(bw))
    want = bw[:, None].double().numpy() * base.double().numpy()
    for r in range(rows):
        for k in range(top):
            e = int(ids[r, k])
            m = gu[e].double().numpy()
            want[r] += float(p[r, k]) * plain.gated_ff(x[r].double().numpy(), m[:ff], m[ff:], down[e].double().numpy())
    tol = 2e-5 if dtype == torch.float32 else 3e-2
    assert np.abs(out.float().cpu().numpy() - want).max() <= tol * max(1.0, np.abs(want).max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("group, ff", [(0, 40), (8, 40), (0, 13)])
def test_silu_activation_of_expert_rows(group, ff, dtype):
    from strata_inference_b200.kernels import native
    g = torch.Generator().manual_seed(ff)
    gate, up = (torch.randn((9, ff), generator=g).to(dtype).float() for _ in range(2))
    if group:
        gu = torch.stack([gate.view(9, -1, 8), up.view(9, -1, 8)], dim=2).reshape(9, 2 * ff)
    else:
        gu = torch.cat([gate, up], dim=1)
    y = torch.empty((9, ff), dtype=dtype, device="cuda")
    native.expert_activate(_dev(gu, dtype), y, None, 0.0, 0.0, native.FORM_GATED_SILU, group)
    want = plain.silu(gate.double().numpy()) * up.double().numpy()
    assert np.abs(y.float().cpu().numpy() - want).max() <= (1e-5 if dtype == torch.float32 else 3e-2)


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


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width, taps", [(64, 4), (72, 2), (33, 5), (256, 1), (1032, 3), (20, 9)])
def test_short_convolution_alone(width, taps, dtype):
    """Two sequences in portions (down to one row, some shorter than the reach, one beside a filler
    without a slot) against the plain convolution of the whole sequences."""
    from strata_inference_b200.kernels import native
    g = torch.Generator().manual_seed(width)
    w = torch.randn((width, taps), generator=g)
    xs = [torch.randn((40, width), generator=g).to(dtype).float() for _ in range(2)]
    refs = [x.double().numpy() + plain.causal_conv(x.double().numpy(), w.double().numpy()) for x in xs]
    state = torch.full((3, max(1, -(-(taps - 1) * width // 4) * 4)), 5.0, device="cuda")
    state[[0, 2]] = 0.0
    d_w, at = _dev(w.t()), [0, 0]
    for counts in ((7, 1), (1, 1), (2, 3), (1, 1), (1, 1), (1, 0), (13, 20), (0, 1), (1, 1)):
        live = [b for b in range(2) if counts[b]]
        seqs = [((2, 0)[b], at[b], counts[b]) for b in live]
        x = [xs[b][at[b]:at[b] + counts[b]] for b in live]
        if counts == (2, 3):
            seqs.append((-1, 0, 4))
            x.append(torch.ones((4, width)))
        ctx = _Step(seqs)
        y = torch.empty((ctx.n_rows, width), dtype=dtype, device="cuda")
        native.short_conv(_dev(torch.cat(x), dtype), y, d_w, state, ctx)
        row = 0
        for b in live:
            want = refs[b][at[b]:at[b] + counts[b]]
            got = y[row:row + counts[b]].float().cpu().numpy()
            assert np.abs(got - want).max() <= (2e-5 if dtype == torch.float32 else 3e-2) * np.abs(want).max(), (counts, b)
            at[b] += counts[b]
            row += counts[b]
    assert float((state[1] - 5.0).abs().max()) == 0.0, "a slot that no sequence of the step holds is left alone"


@pytest.mark.parametrize("width, taps", [(64, 4), (264, 2), (1032, 3), (256, 1), (128, 6), (4608, 4)])
def test_residual_step_with_the_convolution(width, taps):
    """h += rms(a) post, y = x + conv(x) with x = rms(h) pre, one row per sequence over several steps,
    against the two launches it stands for (bit for bit) and the plain formulas."""
    from strata_inference_b200.kernels import native
    assert native.add_norm_conv_supports(width)
    g = torch.Generator().manual_seed(width + taps)
    w = torch.randn((taps, width), generator=g).cuda()
    post, pre = (torch.randn(width, generator=g).cuda() for _ in range(2))
    n_state = max(1, -(-(taps - 1) * width // 4) * 4)
    state, other = torch.zeros((4, n_state), device="cuda"), torch.zeros((4, n_state), device="cuda")
    seen = {0: [], 3: []}
    for step in range(5):
        seqs = [(3, step, 1), (-1, 0, 1), (0, step, 1)]
        ctx = _Step(seqs)
        a = torch.randn((3, width), generator=g).to(torch.bfloat16).cuda()
        h = torch.randn((3, width), generator=g).cuda()
        h2, x = h.clone(), torch.empty_like(a)
        y, y2 = torch.empty_like(a), torch.empty_like(a)
        pg = post if step % 2 else None
        native.add_norm_conv(a, pg, 1e-5, h, pre, 1e-6, w, state, y, ctx)
        native.add_rms_norm(a, pg, 1e-5, h2, pre, 1e-6, x)
        native.short_conv(x, y2, w, other, ctx)
        assert (h - h2).abs().max() <= 1e-5 and (y.float() - y2.float()).abs().max() <= 3e-2 * y2.float().abs().max()
        for k, slot in enumerate((3, None, 0)):
            if slot is not None:
                seen[slot].append(x[k].double().cpu().numpy())
                hist = np.stack(seen[slot])
                want = hist[-1] + plain.causal_conv(hist, w.t().double().cpu().numpy())[-1]
                assert np.abs(y[k].double().cpu().numpy() - want).max() <= 3e-2 * np.abs(want).max()
    assert (state - other).abs().max() <= 2e-2 * max(1.0, other.abs().max().item())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads, kv, kd, vd, rot, style, rows", [
    (3, 1, 24, 16, 24, 1, 5), (4, 2, 64, 64, 64, 1, 7), (4, 2, 128, 128, 64, 1, 70), (2, 1, 256, 256, 8, 1, 130),
    (4, 4, 64, 64, 0, 0, 9), (2, 2, 20, 30, 10, 0, 66), (8, 1, 64, 64, 16, 1, 200), (4, 2, 64, 64, 6, 1, 80)])
def test_heads_prepared_with_the_norm_behind_the_rotation(heads, kv, kd, vd, rot, style, rows, dtype):
    """Rotation with a magnitude, then the root mean square, then the head's factor; keys and values
    also in the cells of a ring that begins behind fixed cells, older rows of the step left out."""
    from strata_inference_b200.kernels import native
    g = torch.Generator().manual_seed(kd + rows)
    pad = -(-max(kd, vd) // 16) * 16
    proj = torch.randn((rows, heads * kd + kv * (kd + vd)), generator=g).to(dtype).float()
    temp = torch.randn(heads, generator=g)
    freqs = [0.9 * 0.7 ** i for i in range(rot // 2)]
    page, fixed, ring, start = 16, 32, 48, 20
    pos = np.arange(start, start + rows)
    end = start + rows
    qkv = torch.full((rows, (heads + 2 * kv) * pad), float("nan"), dtype=dtype, device="cuda")
    kp, vp = (torch.full((9, kv, page, pad), -7.0, dtype=dtype, device="cuda") for _ in range(2))
    table = torch.zeros((2, 5), dtype=torch.int32)
    table[1] = torch.tensor([6, 1, 8, 3, 5])
    native.head_prepare(_dev(proj, dtype), qkv, None, None, None, 1e-5, _dev(torch.tensor(freqs)) if rot else None, rot,
                        None, None, i32(pos.tolist()), i32([0] * rows), i32([1]), i32([end]), kp, vp, table.cuda(), page,
                        ring, heads, kv, kd, vd, pad, style=style, norm_after=True, temp=_dev(temp), magnitude=1.3,
                        fixed_tokens=fixed)
    p = proj.double().numpy()
    q = p[:, :heads * kd].reshape(rows, heads, kd)
    k = p[:, heads * kd:(heads + kv) * kd].reshape(rows, kv, kd)
    v = p[:, (heads + kv) * kd:].reshape(rows, kv, vd)

    def turned(x):
        if style == 1:
            return plain.rotate_pairs(x, pos, rot, freqs, 1.3)
        y = x.copy()                             # half-split pairs (i, i + rot / 2)
        for i in range(rot // 2):
            c, s = (1.3 * np.cos(pos * freqs[i]))[:, None], (1.3 * np.sin(pos * freqs[i]))[:, None]
            u, w = x[..., i], x[..., i + rot // 2]
            y[..., i], y[..., i + rot // 2] = u * c - w * s, w * c + u * s
        return y
    q = plain.unit_rms(turned(q), 1e-5) * temp.double().numpy()[:, None]
    k = plain.unit_rms(turned(k), 1e-5)
    want = np.zeros((rows, heads + 2 * kv, pad))
    want[:, :heads, :kd], want[:, heads:heads + kv, :kd], want[:, heads + kv:, :vd] = q, k, v
    tol = 5e-5 if dtype == torch.float32 else 2e-2
    got = qkv.float().cpu().numpy().reshape(rows, heads + 2 * kv, pad)
    assert np.abs(got - want).max() <= tol * np.abs(want).max()
    kc, vc = kp.float().cpu().numpy(), vp.float().cpu().numpy()
    held = set()
    for r, t in enumerate(pos):
        if t >= fixed and t < end - ring:
            continue                             # (a later row owns the cell)
        cell = t if t < fixed else fixed + (t - fixed) % ring
        held.add(cell)
        pg = int(table[1, cell // page])
        assert np.abs(kc[pg, :, cell % page] - got[r, heads:heads + kv]).max() == 0.0
        assert np.abs(vc[pg, :, cell % page] - got[r, heads + kv:]).max() == 0.0
    free = [c for c in range(80) if c not in held]
    for c in free:
        assert (kc[int(table[1, c // page]), :, c % page] == -7.0).all()


def _kept_reference(q, k, v, scale, window, keep, rows=None):
    """q[T, H, d], k and v [T, G, d] of one sequence: rows of a 64-bit softmax over the window and
    the kept first positions."""
    T, H, d = q.shape
    G = k.shape[1]
    q, k, v = (x.double().numpy() for x in (q, k, v))
    out = np.zeros((T, H, d))
    for t in range(T) if rows is None else rows:
        seen = plain.visible(t, window, keep)
        for a in range(H):
            out[t, a] = plain.softmax((k[seen, a // (H // G)] @ q[t, a]) * scale) @ v[seen, a // (H // G)]
    return out


def _paged_ring(k, v, page, fixed, ring, dtype, g):
    """Keys and values of one sequence as the cache holds them after its last position, pages in
    any order; cells that hold nothing are loud."""
    T, kv, d = k.shape
    cells = fixed + ring if ring else -(-T // page) * page
    n_pages = cells // page
    order = torch.randperm(n_pages + 3, generator=g)[:n_pages]
    kp = torch.full((n_pages + 3, kv, page, d), 1e4, dtype=dtype)
    vp = torch.full((n_pages + 3, kv, page, d), 1e4, dtype=dtype)
    for t in range(T):
        if ring and fixed <= t < T - ring:
            continue
        c = fixed + (t - fixed) % ring if ring and t >= fixed else t
        kp[order[c // page], :, c % page], vp[order[c // page], :, c % page] = k[t].to(dtype), v[t].to(dtype)
    table = torch.zeros((2, n_pages), dtype=torch.int32)
    table[1] = order.to(torch.int32)
    return kp.cuda(), vp.cuda(), table.cuda()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("window, keep, heads, kv, hd, splits", [(7, 3, 4, 2, 16, 1), (40, 20, 6, 1, 48, 3), (64, 70, 2, 2, 64, 5),
                                                                (1, 5, 2, 1, 32, 2), (500, 9, 3, 3, 16, 4)])
def test_general_attention_kernel_with_kept_positions(window, keep, heads, kv, hd, splits, dtype):
    """Prompt rows of two sequences over their packed keys, then the last rows of one over a ring
    behind fixed cells, cut into runs."""
    from strata_inference_b200.kernels import native
    g = torch.Generator().manual_seed(window + keep)
    lens = [230, 37]
    R = sum(lens)
    q = torch.randn((R, heads, hd), generator=g).to(dtype).float()
    k, v = (torch.randn((R, kv, hd), generator=g).to(dtype).float() for _ in range(2))
    d_qkv = _dev(torch.cat([x.reshape(R, -1) for x in (q, k, v)], dim=1), dtype)
    ctx = _Step([(0, 0, lens[0]), (1, 0, lens[1])])
    out = torch.empty((R, heads * hd), dtype=dtype, device="cuda")
    width = d_qkv.shape[1]
    native.attention_rows(d_qkv, width, d_qkv[:, heads * hd:], d_qkv[:, (heads + kv) * hd:], width, None, None, None,
                          64, 0, ctx.row_pos, ctx.row_seq, ctx.seq_slot, ctx.seq_start, ctx.seq_row0, out, None, heads, kv,
                          hd, 0.4, 0.0, window, 1, keep=keep)
    ref = np.concatenate([_kept_reference(q[a:b], k[a:b], v[a:b], 0.4, window, keep) for a, b in ((0, 230), (230, R))])
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    assert np.abs(out.float().cpu().numpy().reshape(R, heads, hd) - ref).max() <= tol
    page, T = 16, lens[0]
    fixed = -(-keep // page) * page
    ring = -(-(window + 15) // page) * page
    if fixed + ring >= T:
        fixed = ring = 0
    kp, vp, table = _paged_ring(k[:T], v[:T], page, fixed, ring, dtype, g)
    n = 9
    step = _Step([(1, T - n, n)])
    out = torch.empty((n, heads * hd), dtype=dtype, device="cuda")
    qs = _dev(q[T - n:T].reshape(n, -1), dtype)
    scratch = torch.empty(native.attention_rows_scratch_bytes(n, heads, hd, splits) + 16, dtype=torch.uint8, device="cuda")
    native.attention_rows(qs, heads * hd, None, None, heads * hd, kp, vp, table, page, ring, step.row_pos, step.row_seq,
                          step.seq_slot, step.seq_start, step.seq_row0, out, scratch, heads, kv, hd, 0.4, 0.0, window, splits,
                          keep=keep, fixed_tokens=fixed)
    assert np.abs(out.float().cpu().numpy().reshape(n, heads, hd) - ref[T - n:T]).max() <= tol


@pytest.mark.parametrize("nh, nkv, hd, window, keep, splits, warps", [
    (4, 2, 128, 96, 20, 1, 4), (4, 2, 128, 96, 20, 3, 4), (8, 1, 64, 40, 70, 5, 2), (2, 2, 256, 16, 1, 2, 8),
    (8, 4, 256, 100, 33, 20, 4), (16, 2, 64, 7, 16, 1, 1), (4, 4, 128, 1, 17, 2, 4), (8, 2, 128, 1000, 50, 40, 8),
    (2, 1, 128, 33, 15, 70, 8), (4, 2, 64, 30, 100, 6, 8), (2, 1, 64, 15, 5, 3, 2)])
def test_decode_kernel_with_kept_positions(nh, nkv, hd, window, keep, splits, warps):
    """The bfloat16 decode kernel over a ring behind fixed cells, pages in any order: positions where
    the window leaves the kept tokens, at tile, page and ring borders; every way of joining the runs."""
    from strata_inference_b200.kernels import native
    assert native.attention_decode_supports(nh, nkv, hd, 16)
    g = torch.Generator().manual_seed(nh * hd + window)
    page, scale = 16, 3.0 / math.sqrt(hd)
    top = 330
    q = torch.randn((top, nh, hd), generator=g).to(torch.bfloat16)
    k, v = (torch.randn((top, nkv, hd), generator=g).to(torch.bfloat16) for _ in range(2))
    fixed = -(-keep // page) * page
    ring = -(-(window + 15) // page) * page
    ends = sorted({1, 2, 16, 17, keep, keep + 1, window, window + 1, window + keep - 1, window + keep, window + keep + 1,
                   fixed + ring, fixed + ring + 1, fixed + ring + 17, top - 1, top})
    for T in [e for e in ends if 0 < e <= top]:
        f, r = (fixed, ring) if fixed + ring < T else (0, 0)
        kp, vp, table = _paged_ring(k[:T], v[:T], page, f, r, torch.bfloat16, g)
        ref = _kept_reference(q[:T], k[:T], v[:T], scale, window, keep, rows=[T - 1])[T - 1]
        out = torch.empty((1, nh * hd), dtype=torch.bfloat16, device="cuda")
        scratch = torch.empty(max(16, native.attention_rows_scratch_bytes(1, nh, hd, splits)), dtype=torch.uint8, device="cuda")
        tickets = torch.zeros(nkv, dtype=torch.int32, device="cuda")
        native.attention_decode(q[T - 1].reshape(1, -1).contiguous().cuda(), nh * hd, kp, vp, table, page, r, i32([T - 1]),
                                i32([0]), i32([1]), out, scratch, tickets, nh, nkv, hd, scale, 0.0, window, splits, warps,
                                fresh=1, keep=keep, fixed_tokens=f)
        assert int(tickets.abs().sum()) == 0, "the ticket counters are put back"
        err = np.abs(out.float().cpu().numpy().reshape(nh, hd) - ref).max()
        assert err <= 2e-2 * max(1.0, np.abs(ref).max()), f"{T} positions: {err:.3e}"


@pytest.mark.parametrize("heads, kv, hd, window, keep, lens", [
    (4, 2, 128, 96, 20, [398, 23, 97]), (4, 4, 64, 40, 70, [300, 5, 64, 131]), (2, 1, 256, 128, 1, [700, 130]),
    (4, 2, 64, 1, 200, [500]), (2, 2, 128, 5000, 50, [600]), (4, 2, 128, 200, 128, [900, 300]), (2, 1, 64, 33, 129, [400, 128])])
def test_prompt_kernels_with_kept_positions(heads, kv, hd, window, keep, lens):
    """The tcgen05 prompt kernel (as a grid and as a balanced list, split or not) and the mma.sync one
    against the 64-bit softmax over window and kept positions; then the last rows of every sequence
    with the rows before them as keys only."""
    from strata_inference_b200.kernels import native
    assert native.attention_prefill_tc_supports(heads, kv, hd, (heads + 2 * kv) * hd)
    g = torch.Generator().manual_seed(heads + hd + window)
    scale = 3.0 / math.sqrt(hd)
    rows, refs, row0, at = [], [], [], 0
    for T in lens:
        q = torch.randn((T, heads, hd), generator=g).to(torch.bfloat16)
        k, v = (torch.randn((T, kv, hd), generator=g).to(torch.bfloat16) for _ in range(2))
        refs.append(_kept_reference(q, k, v, scale, window, keep))
        rows.append(torch.cat([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], dim=1))
        row0.append(at)
        at += T
    packed = torch.cat(rows).contiguous().cuda()
    ref = np.concatenate(refs).reshape(at, -1)

    def check(out, what, start=None):
        got = out.float().cpu().numpy()
        for b, T in enumerate(lens):
            lo = row0[b] + (start[b] if start else 0)
            err = np.abs(got[lo:row0[b] + T] - ref[lo:row0[b] + T]).max()
            assert err <= 2e-2 * np.abs(ref).max(), f"{what}, sequence {b}: {err:.3e} of {np.abs(ref).max():.3e}"

    def run(host, start=None):
        out = torch.full((at, heads * hd), float("nan"), dtype=torch.bfloat16, device="cuda")
        if host:
            items, need, n_tickets = native.attention_prefill_tc_plan(lens, heads, kv, hd, window, start, keep)
            assert items > 0
        else:
            need, n_tickets = native.attention_prefill_tc_split(len(lens), max(lens), heads, kv, hd)
        native.attention_prefill_tc(packed, out, i32(row0), i32(lens), len(lens), max(lens), heads, kv, hd, scale, 0.0, window,
                                    torch.empty(max(need, 16), dtype=torch.uint8, device="cuda"),
                                    torch.zeros(max(n_tickets, 1), dtype=torch.int32, device="cuda"),
                                    lens if host else None, i32(start) if start else None, start if host else None, keep=keep)
        assert native.attention_prefill_tc_error() == 0
        check(out, f"tcgen05, {'list' if host else 'grid'}, from {start}", start)
    for host in (False, True):
        run(host)
        run(host, [max(0, T - 40) for T in lens])
    if native.attention_prefill_supports(heads, kv, hd):
        out = torch.full((at, heads * hd), float("nan"), dtype=torch.bfloat16, device="cuda")
        native.attention_prefill(packed, out, i32(row0), i32(lens), len(lens), max(lens), heads, kv, hd, scale, 0.0, window, keep)
        check(out, "mma.sync")


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
    w = weights_for(cfg, 21, dtype)
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
    cfg = ALONE["experts_shared"]
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


@pytest.mark.parametrize("rows, top, experts", [(1, 1, 1), (130, 2, 5), (300, 3, 40), (700, 1, 3), (900, 4, 1024)])
def test_pairs_sorted_by_expert(rows, top, experts):
    """Every pair gets a place of its own, experts one after the other; the tiles cover the places,
    none spans two experts or is longer than 256."""
    from strata_inference_b200.kernels import native
    g = torch.Generator().manual_seed(rows)
    # (uneven: low-numbered experts are chosen far more often)
    score = torch.rand((rows, experts), generator=g) ** (1.0 + torch.arange(experts) * 8.0 / experts)
    ids = score.topk(top, dim=1).indices.to(torch.int32)
    where, tiles = native.expert_plan(ids.cuda(), experts)
    where, tiles = where.cpu(), tiles.cpu().tolist()
    assert sorted(where.view(-1).tolist()) == list(range(rows * top))
    by_place = torch.empty(rows * top, dtype=torch.int32)
    by_place[where.view(-1).long()] = ids.view(-1)
    assert (by_place[1:] >= by_place[:-1]).all()
    at = 0
    for k in range(tiles[0]):
        row0, n, e = tiles[1 + 3 * k:4 + 3 * k]
        assert row0 == at and 0 < n <= 256 and (by_place[row0:row0 + n] == e).all()
        at += n
    assert at == rows * top
    x = torch.randn((rows, 20), generator=g).cuda()
    xs = native.spread_rows(x, where.cuda(), torch.empty((rows * top, 20), device="cuda"))
    assert torch.equal(xs[where.view(-1).long().cuda()].view(rows, top, 20), x[:, None].expand(rows, top, 20))


@pytest.mark.parametrize("counts, N, K", [([256, 1, 0, 300], 128, 64), ([5, 700, 0, 0, 33, 257], 200, 136), ([130], 72, 512),
                                          ([0, 40, 40, 40, 600, 12, 90], 384, 256)])
def test_grouped_products(counts, N, K):
    """Sorted rows times their groups' matrices: plain, and gate and up with the SiLU and the clipped
    gate, widths that are and are not whole tiles, groups without a row."""
    from strata_inference_b200.kernels import native
    g = torch.Generator().manual_seed(N)
    ids = torch.cat([torch.full((c,), e, dtype=torch.int32) for e, c in enumerate(counts)])
    where, tiles = native.expert_plan(ids[:, None].cuda(), len(counts))
    x = torch.randn((len(ids), K), generator=g).to(torch.bfloat16)
    w = (torch.randn((len(counts), 2 * N, K), generator=g) / math.sqrt(K)).to(torch.bfloat16)
    ref = torch.stack([w[int(e)].double() @ r for e, r in zip(ids, x.double())])
    out = torch.full((len(ids), 2 * N), float("nan"), dtype=torch.bfloat16, device="cuda")
    native.gemm_tcgen05_grouped(x.cuda(), w.cuda(), tiles, out)
    assert (out.cpu().double() - ref).abs().max() <= 1e-2 * ref.abs().max()
    for epi, cap in ((native.EPI_SWIGLU, 0.0), (native.EPI_CLIPPED, 1.2)):
        a, u = ref[:, :N], ref[:, N:]
        if cap:
            a, u = a.clamp(max=cap), u.clamp(-cap, cap)
            want = a * torch.sigmoid(1.702 * a) * (u + 1.0)
        else:
            want = a * torch.sigmoid(a) * u
        out = torch.full((len(ids), N), float("nan"), dtype=torch.bfloat16, device="cuda")
        native.gemm_tcgen05_grouped(x.cuda(), w.cuda(), tiles, out, epi, cap)
        assert (out.cpu().double() - want).abs().max() <= 1e-2 * want.abs().max()
    assert native.gemm_tcgen05_error() == 0
