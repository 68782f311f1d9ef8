"""Small Simetar configurations for the tests, random weights for them, and the comparison with
the plain model (tests/plain_simetar.py)."""

from __future__ import annotations

import copy
import math
import random
from typing import Dict, List, Sequence

import numpy as np
import torch

import plain_simetar as plain


def dense(ff):
    return {"kind": "dense", "ff": ff}


def llama3(factor=6.0, low=1.0, high=3.0, original=100):
    return {"factor": factor, "low": low, "high": high, "original": original}


def yarn(factor=4.0, original=96, fast=8.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def _rot(dims, base, scaling):
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = scaling
    return rot


def attention(heads, kv_heads, dim, size, conv=3, scale=0.2, softcap=15.0, rot_dims=None, base=10000.0, scaling=None,
              mlp=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "conv": conv, "scale": scale}
    if softcap:
        mixer["softcap"] = softcap
    if rot_dims != 0:
        mixer["rot"] = _rot(dim if rot_dims is None else rot_dims, base, scaling)
    if size:
        mixer["mask"] = {"size": size}
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, rank, scale=0.3, base=10000.0, scaling=None, kv_from=None, mlp=None):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale,
             "rot": _rot(rot_dim, base, scaling)}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


def model(width, vocab, layers, eps=1e-5):
    return {"architecture": "Simetar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": list(layers)}


# one mechanism at a time
ALONE = {
    "open": model(64, 200, [attention(4, 2, 16, 0, conv=1, softcap=0, rot_dims=0)]),
    "conv": model(64, 200, [attention(2, 2, 16, 0, conv=5, rot_dims=0)]),
    "two_taps": model(64, 200, [attention(2, 1, 16, 30, conv=2)]),
    "cap": model(64, 200, [attention(4, 1, 16, 0, conv=1, scale=0.6, softcap=1.5, rot_dims=0)]),
    "rotation": model(64, 200, [attention(4, 4, 16, 0, rot_dims=8, base=500.0)]),
    "llama3": model(64, 200, [attention(4, 2, 24, 0, scaling=llama3())]),
    "llama3_partial": model(64, 200, [attention(3, 1, 32, 0, rot_dims=12, base=300.0, scaling=llama3(9.0, 0.5, 6.0, 60))]),
    "window": model(64, 200, [attention(4, 2, 16, 24)]),
    "dense": model(64, 200, [attention(2, 2, 16, 40, mlp=dense(72))]),
    "latent": model(64, 200, [latent(4, 16, 8, 16, 32)]),
    "latent_yarn": model(64, 200, [latent(3, 20, 12, 10, 24, scaling=yarn(), mlp=dense(40))]),
    "lent": model(64, 200, [latent(2, 16, 8, 16, 24, scaling=yarn()), latent(2, 16, 8, 16, 24, scaling=yarn(), kv_from=0)]),
}

# windows shorter and longer than a page of 64 and none; a lender with two readers whose heads, widths
# and scales differ from its own, another lender between them, layers with and without a feed-forward
MIXED = model(64, 200, [
    attention(4, 2, 16, 37, rot_dims=8, scaling=llama3(), mlp=dense(96)),
    latent(4, 16, 8, 24, 40, scaling=yarn(), mlp=dense(64)),
    attention(3, 1, 32, 90, conv=2, scale=0.15, softcap=8.0),
    latent(2, 24, 8, 16, 40, scale=0.2, scaling=yarn(), kv_from=1),
    latent(3, 16, 4, 8, 24, base=500.0, mlp=dense(40)),
    attention(2, 2, 24, 0, conv=4, base=300.0, softcap=0, mlp=dense(48)),
    latent(5, 12, 8, 20, 40, scale=0.4, scaling=yarn(), kv_from=1, mlp=dense(80)),
    latent(1, 32, 4, 12, 24, base=500.0, kv_from=4),
])

# sizes that are no multiples of 16, 8 or 4; one head; a window of one position
ODD = model(70, 131, [
    attention(3, 3, 10, 7, conv=7, rot_dims=6, scaling=llama3(3.0, 0.7, 4.0, 50), mlp=dense(33)),
    latent(3, 9, 6, 5, 17, scaling=yarn(3.0, 50, 4.0, 0.7), mlp=dense(20)),
    attention(1, 1, 20, 33, conv=1, base=50.0, softcap=4.0),
    attention(5, 1, 6, 1, conv=2, scale=0.5),
    latent(1, 13, 6, 21, 17, scale=0.5, scaling=yarn(3.0, 50, 4.0, 0.7), kv_from=1, mlp=dense(7)),
    attention(3, 1, 13, 50, conv=3, rot_dims=2),
], eps=1e-6)

# heads of the fast kernels' widths (64, 128, 256), groups of 1, 2, 4 and 8, more than 16 latent heads, a
# window of one position and one longer than any request
WIDE = model(128, 300, [
    attention(4, 2, 64, 48, base=500000.0, scale=0.12, scaling=llama3(16.0, 1.0, 4.0, 128), mlp=dense(256)),
    latent(4, 64, 32, 64, 96, scale=0.1, scaling=yarn(16.0, 128, 32.0, 1.0)),
    attention(8, 1, 128, 130, rot_dims=64, scale=0.08, mlp=dense(136)),
    attention(2, 1, 256, 1, conv=2, rot_dims=64, scale=0.06),
    latent(18, 32, 32, 32, 96, scale=0.15, scaling=yarn(16.0, 128, 32.0, 1.0), kv_from=1, mlp=dense(64)),
    attention(4, 1, 64, 5000, conv=4, scale=0.12, softcap=30.0, mlp=dense(128)),
    attention(2, 2, 128, 100, conv=1, scale=0.08, softcap=0, scaling=llama3()),
])

# a scale that makes the softmax pick a few keys among those in sight
SHARP = model(64, 200, [
    attention(4, 2, 16, 50, conv=2, scale=1.0, softcap=40.0, rot_dims=4),
    attention(2, 2, 16, 66, scale=0.9, softcap=40.0, rot_dims=4, mlp=dense(32)),
    latent(2, 16, 4, 16, 24, scale=1.5),
])

REL_TOL = {"float32": 1e-4, "bfloat16": 4e-2}
# A few rows of a random model turn the rounding of activations into an error many times the usual one
# (a sub-layer's output that nearly cancels before its layer norm; the plain model with activations rounded
# to bfloat16 shows the same rows): single rows are bounded loosely, the typical one closely, and the 32-bit
# runs bound every row.
BF16_MEDIAN, BF16_ROWS_OVER, BF16_WORST = 2e-2, 0.1, 0.25


def prompts(cfg: dict, lengths: Sequence[int], seed: int) -> List[List[int]]:
    g = torch.Generator().manual_seed(seed)
    return [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in lengths]


def random_weights(config: dict, seed: int) -> Dict[str, torch.Tensor]:
    """Random tensors of every name the configuration asks for, rounded to bfloat16 values; biases,
    taps and gains large enough that leaving one out, or taking another's, shows."""
    g = torch.Generator().manual_seed(seed)
    W = config["width"]

    def mat(o, i, s=1.0):
        return torch.randn((o, i), generator=g) * (s / math.sqrt(i))

    def vec(n, s=0.3, at=1.0):
        return torch.randn((n,), generator=g) * s + at

    def norm(name):
        out[name], out[name + ".b"] = vec(W), vec(W, 0.3, 0.0)
    out: Dict[str, torch.Tensor] = {"embed": torch.randn((config["vocab"], W), generator=g)}
    for i, layer in enumerate(config["layers"]):
        m, pre = layer["mixer"], f"l{i}.mix."
        H, D = m["heads"], m["dim"]
        norm(f"l{i}.norm1")
        if layer["type"] == "attention":
            for name, n in (("q", H * D), ("k", (m.get("kv_heads") or H) * D)):
                out[pre + name], out[pre + name + ".b"] = mat(n, W), vec(n, 0.4, 0.0)
                out[pre + name + ".conv"] = torch.randn((n, m["conv"]), generator=g) * 0.6
                out[pre + name + ".norm"] = vec(n)
            V = D
        else:
            V, R = m["vdim"], m["kv_rank"]
            out[pre + "q"] = mat(H * (D + m["rot_dim"]), W)
            if m.get("kv_from") is None:
                out[pre + "dkv"], out[pre + "dkv.norm"] = mat(R + m["rot_dim"], W), vec(R)
            out[pre + "uk"], out[pre + "uv"] = mat(H * D, R), mat(H * V, R)
        out[pre + "g"], out[pre + "o"] = mat(H * V, W, 1.5), mat(W, H * V)
        if layer.get("mlp"):
            F, pre = layer["mlp"]["ff"], f"l{i}.mlp."
            norm(f"l{i}.norm2")
            out[pre + "gate"], out[pre + "up"], out[pre + "down"] = mat(F, W), mat(F, W), mat(W, F)
    norm("final.norm")
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
    """A configuration drawn from the design's whole range: both mixers in any order, grouped and
    ungrouped heads of the fast kernels' widths and of others, windows of any length or none, caps or
    none, any number of taps, rotations with and without scaling, readers of earlier layers' rows."""
    r = random.Random(seed)
    width, vocab = r.choice([64, 96, 128, 100, 36]), r.randrange(90, 300)
    layers: list = []
    for i in range(r.randrange(2, 7)):
        mlp = dense(r.choice([8, 24, 40, 130, 33])) if r.random() < 0.75 else None
        lenders = [k for k, l in enumerate(layers) if l["type"] == "latent_attention" and "kv_from" not in l["mixer"]]
        if r.random() < 0.5:
            kv, dim = r.choice([1, 2, 4]), r.choice([16, 32, 64, 64, 128, 24, 10])
            layers.append(attention(
                kv * r.choice([1, 2, 3, 4]), kv, dim, r.choice([0, 1, 5, 16, 37, 64, 100]), conv=r.choice([1, 2, 3, 4, 5, 9]),
                scale=r.choice([0.1, 0.3]), softcap=r.choice([0, 2.0, 20.0, 50.0]), rot_dims=r.choice([0, 2, dim // 4 * 2, dim]),
                base=r.choice([100.0, 10000.0, 500000.0]),
                scaling=r.choice([None, llama3(), llama3(16.0, 1.0, 4.0, 40), llama3(2.0, 2.0, 30.0, 4096)]), mlp=mlp))
            continue
        heads, dim, vdim = r.choice([1, 2, 3, 6, 17]), r.choice([16, 32, 64, 10]), r.choice([16, 48, 64, 7])
        if lenders and r.random() < 0.6:
            k = r.choice(lenders)
            m = layers[k]["mixer"]
            layers.append(latent(heads, dim, m["rot_dim"], vdim, m["kv_rank"], scale=r.choice([0.1, 0.25]), kv_from=k, mlp=mlp))
            layers[-1]["mixer"]["rot"] = dict(m["rot"])
        else:
            layers.append(latent(heads, dim, r.choice([2, 8, 16, 32]), vdim, r.choice([16, 40, 96, 21]), scale=r.choice([0.1, 0.25]),
                                 base=r.choice([100.0, 10000.0]),
                                 scaling=r.choice([None, yarn(), yarn(16.0, 40, 4.0, 0.5), yarn(2.0, 4096, 32.0, 1.0)]), mlp=mlp))
    return model(width, vocab, layers, eps=r.choice([1e-5, 1e-6]))
