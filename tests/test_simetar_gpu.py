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
