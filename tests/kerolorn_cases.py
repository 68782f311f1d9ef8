"""Small Kerolorn configurations for the tests, random weights for them, and the comparison with
the plain model (tests/plain_kerolorn.py)."""

from __future__ import annotations

import copy
import math
import random
from typing import Dict, List, Sequence

import numpy as np
import torch

import plain_kerolorn as plain


def moe(experts, top, ff, shared=0, scale=1.7):
    out = {"kind": "moe", "router": {"experts": experts, "top": top, "scale": scale}, "expert": {"ff": ff}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def yarn(factor=4.0, original=96, fast=8.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def attention(heads, kv_heads, dim, vdim, size, keep=0, scale=0.2, rot_dims=None, base=10000.0, scaling=None, mlp=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot_dims != 0:
        mixer["rot"] = {"base": base, "dims": dim if rot_dims is None else rot_dims}
        if scaling:
            mixer["rot"]["scaling"] = scaling
    if size:
        mixer["mask"] = {"size": size, "keep_first": keep}
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def model(width, vocab, layers, eps=1e-5, taps=3, logit_scale=0.5):
    return {"architecture": "Kerolorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "canon": {"taps": taps},
            "logit_scale": logit_scale, "layers": list(layers)}


# one mechanism at a time
ALONE = {
    "open": model(64, 200, [attention(4, 2, 16, 16, 0, rot_dims=0)], taps=1),
    "conv": model(64, 200, [attention(2, 2, 16, 16, 0, rot_dims=0)], taps=5),
    "two_taps": model(64, 200, [attention(2, 1, 16, 16, 30, 4)], taps=2),
    "rotation": model(64, 200, [attention(4, 4, 16, 24, 0, rot_dims=8, base=500.0)]),
    "yarn": model(64, 200, [attention(4, 2, 24, 16, 0, scaling=yarn())]),
    "yarn_partial": model(64, 200, [attention(3, 1, 32, 32, 0, rot_dims=12, scaling=yarn(8.0, 64, 16.0, 0.5))]),
    "window": model(64, 200, [attention(4, 2, 16, 16, 24)]),
    "kept": model(64, 200, [attention(4, 2, 16, 16, 24, 10)]),
    "kept_pages": model(64, 200, [attention(2, 1, 32, 32, 20, 70, rot_dims=8)]),
    "experts": model(64, 200, [attention(2, 2, 16, 16, 40, 3, mlp=moe(6, 3, 20))]),
    "experts_shared": model(64, 200, [attention(2, 2, 16, 16, 50, mlp=moe(5, 1, 12, shared=28, scale=2.5))], logit_scale=2.0),
}

# windows shorter and longer than a page of 64, kept tokens fewer and more than the window, a layer
# without a mask, values wider and narrower than keys, layers with and without a feed-forward
MIXED = model(64, 200, [
    attention(4, 2, 16, 16, 37, 12, rot_dims=8, scaling=yarn(), mlp=moe(6, 2, 24, shared=32)),
    attention(3, 1, 32, 48, 90, 5, scale=0.15, mlp=moe(4, 1, 32)),
    attention(4, 2, 16, 16, 0, rot_dims=8, scaling=yarn(2.0, 200, 20.0, 2.0), mlp=moe(8, 3, 16, shared=16, scale=0.8)),
    attention(2, 2, 24, 8, 16, 66, base=300.0),
    attention(4, 4, 16, 16, 70, rot_dims=0, mlp=moe(5, 2, 24, shared=40)),
], taps=4)

# sizes that are no multiples of 16, 8 or 4; one head; a top as large as the number of experts
ODD = model(70, 131, [
    attention(3, 3, 10, 14, 7, 3, rot_dims=6, scaling=yarn(3.0, 50, 4.0, 0.7), mlp=moe(3, 3, 10)),
    attention(1, 1, 20, 7, 33, 1, base=50.0, mlp=moe(7, 2, 9, shared=5)),
    attention(5, 1, 6, 9, 1, 2, scale=0.5),
    attention(3, 1, 13, 5, 50, 100, rot_dims=2, mlp=moe(2, 1, 36, shared=36, scale=1.0)),
], eps=1e-6, taps=7, logit_scale=1.0)

# heads of the fast kernels' widths (64, 128, 256), groups of 1, 2, 4 and 8, a window of one position and
# one longer than any request
WIDE = model(128, 300, [
    attention(4, 2, 64, 64, 48, 20, base=500000.0, scale=0.12, scaling=yarn(16.0, 128, 32.0, 1.0), mlp=moe(4, 2, 64, shared=64)),
    attention(8, 1, 128, 128, 130, 70, rot_dims=64, scale=0.08, mlp=moe(3, 1, 40)),
    attention(2, 1, 256, 256, 1, 5, rot_dims=64, scale=0.06),
    attention(4, 1, 64, 64, 5000, 9, scale=0.12, mlp=moe(9, 4, 24, shared=128)),
    attention(2, 2, 128, 128, 100, 64, scale=0.08, scaling=yarn()),
])

# a scale that makes the softmax pick a few keys among those in sight
SHARP = model(64, 200, [
    attention(4, 2, 16, 16, 50, 9, scale=1.0, rot_dims=4),
    attention(2, 2, 16, 24, 66, 17, scale=0.9, rot_dims=4, mlp=moe(3, 1, 32)),
], taps=2)

REL_TOL = {"float32": 1e-4, "bfloat16": 4e-2}
# bfloat16 runs of whole models take weights whose corrections alone choose the experts: a router's
# close call sends a row to another expert, and (through the kept tokens) every later row to other
# keys, which is a different function, not a rounding error.
BF16_MEDIAN, BF16_ROWS_OVER, BF16_WORST = 2e-2, 0.1, 0.12


def prompts(cfg: dict, lengths: Sequence[int], seed: int) -> List[List[int]]:
    g = torch.Generator().manual_seed(seed)
    return [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in lengths]


def random_weights(config: dict, seed: int, decisive: bool = False) -> Dict[str, torch.Tensor]:
    """Random tensors of every name the configuration asks for, rounded to bfloat16 values.  The
    corrections are of the size of the scores' differences, so that they change choices;
    ``decisive``: they lie so far apart that they alone choose, whatever the scores' rounding."""
    g = torch.Generator().manual_seed(seed)
    W = config["width"]

    def mat(o, i, s=1.0):
        return torch.randn((o, i), generator=g) * (s / math.sqrt(i))

    def vec(n, s=0.3, at=1.0):
        return torch.randn((n,), generator=g) * s + at

    out: Dict[str, torch.Tensor] = {"embed": torch.randn((config["vocab"], W), generator=g)}
    for i, layer in enumerate(config["layers"]):
        m, pre = layer["mixer"], f"l{i}.mix."
        H, D, V = m["heads"], m["dim"], m["vdim"]
        G = m.get("kv_heads") or H
        out[f"l{i}.norm1"], out[f"l{i}.norm1b"] = vec(W), vec(W)
        out[f"l{i}.canon1"] = torch.randn((W, config["canon"]["taps"]), generator=g) * 0.5
        out[pre + "q"], out[pre + "k"], out[pre + "v"] = mat(H * D, W), mat(G * D, W), mat(G * V, W)
        out[pre + "temp"] = vec(H, 0.4)
        out[pre + "o"] = mat(W, H * V)
        mlp = layer.get("mlp")
        if not mlp:
            continue
        out[f"l{i}.norm2"], out[f"l{i}.norm2b"] = vec(W), vec(W)
        pre = f"l{i}.mlp."
        E, F = mlp["router"]["experts"], mlp["expert"]["ff"]
        out[pre + "router"] = mat(E, W, 4.0)
        out[pre + "correction"] = torch.randperm(E, generator=g) * 1.5 if decisive else vec(E, 0.3, 0.0)
        for e in range(E):
            out[pre + f"e{e}.gate"], out[pre + f"e{e}.up"], out[pre + f"e{e}.down"] = mat(F, W, 1.5), mat(F, W, 1.5), mat(W, F)
        if mlp.get("shared"):
            S = mlp["shared"]["ff"]
            out[pre + "shared.gate"], out[pre + "shared.up"], out[pre + "shared.down"] = mat(S, W), mat(S, W), mat(W, S)
            out[pre + "shared.sg"] = mat(1, W, 2.0)
    out["final.norm"] = vec(W)
    out["head"] = mat(config["vocab"], W, 2.0)
    return {n: t.to(torch.bfloat16).to(torch.float32) for n, t in out.items()}


def plain_logits(cfg: dict, weights: Dict[str, torch.Tensor], tokens: Sequence[int]) -> torch.Tensor:
    return torch.from_numpy(np.ascontiguousarray(plain.logits(cfg, weights, list(tokens))))


def assert_close(got: torch.Tensor, ref: torch.Tensor, dtype: str, what: str) -> None:
    """Rows of logits against the plain model's: the largest difference as a fraction of the
    largest plain logit of the compared rows."""
    got = got.detach().to("cpu", torch.float64)
    ref = ref.to(torch.float64)
    assert got.shape == ref.shape, f"{what}: shape {tuple(got.shape)} vs {tuple(ref.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite logits"
    scale = ref.abs().max().item()
    diff = (got - ref).abs().amax(dim=-1)
    bad = (diff > REL_TOL[dtype] * scale).nonzero()
    text = (f"{what}: max |diff| {diff.max().item():.3e}, median {diff.median().item():.3e}, "
            f"{bad.numel()} of {got.shape[0]} rows over {REL_TOL[dtype]:.0e} x max|ref| {scale:.3e}"
            + (f"; first of them row {int(bad[0])}" if bad.numel() else ""))
    if dtype == "float32":
        assert bad.numel() == 0, text
    elif got.shape[0] < 8:
        assert diff.max().item() <= BF16_WORST * scale, text
    else:
        assert diff.median().item() <= BF16_MEDIAN * scale, text
        assert bad.numel() <= max(1, BF16_ROWS_OVER * got.shape[0]), text
        assert diff.max().item() <= BF16_WORST * scale, text


def rows_that_differ(a: torch.Tensor, b: torch.Tensor, factor: float = 100.0) -> int:
    """How many rows of two plain results differ by more than ``factor`` times the 32-bit
    tolerance: what a test needs to be able to tell the two apart."""
    scale = a.abs().max().item()
    return int(((a - b).abs().amax(dim=-1) > factor * REL_TOL["float32"] * scale).sum())


def changed(cfg: dict, edit) -> dict:
    other = copy.deepcopy(cfg)
    edit(other)
    return other


def random_model(seed: int) -> dict:
    """A configuration drawn from the design's whole range: grouped and ungrouped heads of the fast
    kernels' widths and of others, values wider and narrower than keys, any rotation or none, windows of
    any length or none, any number of kept tokens, any number of taps, experts or no feed-forward."""
    r = random.Random(seed)
    width, vocab = r.choice([64, 96, 128, 100, 36]), r.randrange(90, 300)
    layers = []
    for _ in range(r.randrange(2, 6)):
        mlp = None
        if r.random() < 0.75:
            experts = r.randrange(1, 10)
            mlp = moe(experts, r.randrange(1, min(experts, 4) + 1), r.choice([8, 24, 40]), r.choice([0, 16, 36]),
                      scale=r.choice([0.5, 1.0, 3.0]))
        kv = r.choice([1, 2, 4])
        dim = r.choice([16, 32, 64, 64, 128, 24, 10])
        size = r.choice([0, 1, 5, 16, 37, 64, 100])
        layers.append(attention(
            kv * r.choice([1, 2, 3, 4]), kv, dim, r.choice([dim, dim, dim, 16, 48, 128]), size, r.choice([0, 1, 4, 20, 64, 90]),
            scale=r.choice([0.1, 0.3]), rot_dims=r.choice([0, 2, dim // 4 * 2, dim]), base=r.choice([100.0, 10000.0, 500000.0]),
            scaling=r.choice([None, yarn(), yarn(16.0, 40, 4.0, 0.5), yarn(2.0, 4096, 32.0, 1.0)]), mlp=mlp))
    return model(width, vocab, layers, eps=r.choice([1e-5, 1e-6]), taps=r.choice([1, 2, 3, 4, 5, 9]),
                 logit_scale=r.choice([0.25, 1.0, 1.5]))
