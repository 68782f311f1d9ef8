"""A plain, slow Kerolorn in 64-bit numpy: one function per mechanism, whole sequences only.

Nothing here is shared with the package: no cache, no state, no steps, no kernels.  A
sequence is worked on as a whole, every position from the sequence's first token, so that
what the package does with pages, rings, slots, convolution histories and recorded steps has
something independent to be compared with.

Notation: n tokens, width W; x[t] is row t.  Weights are stored [out, in] and applied as
W x.  ``w`` of a function: the tensors of that part by their short names.
"""

from __future__ import annotations

import math

import numpy as np


def f64(t) -> np.ndarray:
    """A stored tensor (torch or numpy, any type) as 64-bit numpy."""
    if hasattr(t, "detach"):
        t = t.detach().to("cpu").double().numpy()
    return np.asarray(t, dtype=np.float64)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def unit_rms(x, eps):
    """Rows of the last axis divided by their root mean square (eps inside the root)."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def causal_conv(h, w):
    """h[n, W], w[W, taps]: per channel the sum over the last ``taps`` rows, the row itself with
    the last tap; rows before the sequence's start are zeros."""
    n, taps = h.shape[0], w.shape[1]
    out = np.zeros_like(h)
    for t in range(n):
        for j in range(taps):
            at = t - taps + 1 + j
            if at >= 0:
                out[t] += w[:, j] * h[at]
    return out


def yarn_frequencies(dims, base, scaling):
    """(frequencies of the dims / 2 pairs, factor on cosine and sine).  Without ``scaling``:
    base^(-2i/dims) and 1.  With it, pairs that turn often within ``original`` positions keep
    their frequency, pairs that turn rarely are slowed down by ``factor``, and a straight ramp
    over the pair's index lies between."""
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return plain, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def index_of(turns):
        # the (real) pair index whose frequency makes that many turns in `original` positions
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(index_of(scaling["fast"])), 0)
    hi = min(math.ceil(index_of(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = (i - lo) / max(hi - lo, 0.001)
        ramp = min(max(ramp, 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate_pairs(x, positions, dims, freqs, magnitude):
    """Rotary positions on the first ``dims`` entries of the last axis of x[n, heads, d]: entry
    2i is paired with entry 2i + 1; the pair's angle at position p is p freqs[i], cosine and
    sine are both multiplied by ``magnitude``.  What lies behind ``dims`` passes unchanged."""
    y = x.copy()
    p = np.asarray(positions, dtype=np.float64)
    for i in range(dims // 2):
        ang = p * freqs[i]
        c, s = (magnitude * np.cos(ang))[:, None], (magnitude * np.sin(ang))[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = u * c - v * s
        y[..., 2 * i + 1] = v * c + u * s
    return y


def visible(t, size, keep):
    """The positions that position t sees: the last ``size`` (its own included; 0: all earlier
    ones) and the sequence's first ``keep``."""
    return [j for j in range(t + 1) if not size or t - j < size or j < keep]


def softmax(s):
    e = np.exp(s - s.max())
    return e / e.sum()


def attention(h, w, m, eps):
    """h[n, W] -> [n, W].  Grouped heads; q and k are rotated, then divided by their root mean
    square per head; a score is (q . k) scale temp_h; a window that also keeps the first
    tokens."""
    n = h.shape[0]
    H, d, vd = m["heads"], m["dim"], m["vdim"]
    G = m.get("kv_heads") or H
    q = (h @ w["q"].T).reshape(n, H, d)
    k = (h @ w["k"].T).reshape(n, G, d)
    v = (h @ w["v"].T).reshape(n, G, vd)
    if m.get("rot"):
        rot = m["rot"]
        freqs, mag = yarn_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
        q = rotate_pairs(q, np.arange(n), rot["dims"], freqs, mag)
        k = rotate_pairs(k, np.arange(n), rot["dims"], freqs, mag)
    q, k = unit_rms(q, eps), unit_rms(k, eps)
    mask = m.get("mask") or {}
    size, keep = mask.get("size") or 0, mask.get("keep_first") or 0
    out = np.zeros((n, H, vd))
    for t in range(n):
        seen = visible(t, size, keep)
        for a in range(H):
            g = a // (H // G)
            s = (k[seen, g] @ q[t, a]) * m["scale"] * w["temp"][a]
            out[t, a] = softmax(s) @ v[seen, g]
    return out.reshape(n, H * vd) @ w["o"].T


def gated_ff(h, gate, up, down):
    """W_down (silu(W_gate h) * (W_up h))."""
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def router_choice(h, w, mlp):
    """(chosen experts [n, top], their weights [n, top]).  Scores softmax over all experts;
    scores plus the correction choose (ties: the lower index); the weights are the scores
    without it, times ``scale``, whatever they sum to."""
    r = mlp["router"]
    z = h @ w["router"].T
    ids, ps = [], []
    for t in range(h.shape[0]):
        s = softmax(z[t])
        chosen = np.argsort(-(s + w["correction"]), kind="stable")[:r["top"]]
        ids.append(chosen)
        ps.append(s[chosen] * r["scale"])
    return np.array(ids), np.array(ps)


def routed_ff(h, w, mlp):
    ids, ps = router_choice(h, w, mlp)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in zip(ids[t], ps[t]):
            out[t] += p * gated_ff(h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"])
    if mlp.get("shared"):
        one = gated_ff(h, w["shared.gate"], w["shared.up"], w["shared.down"])
        out += sigmoid(h @ w["shared.sg"].T) * one
    return out


def sub(weights, prefix):
    return {k[len(prefix):]: f64(v) for k, v in weights.items() if k.startswith(prefix)}


def layer_streams(config, weights, tokens):
    """The residual stream after every layer, [layers, n, W]."""
    eps = config["norm"]["eps"]
    x = f64(weights["embed"])[np.asarray(tokens, dtype=np.int64)]
    out = []
    for i, layer in enumerate(config["layers"]):
        h = rms_norm(x, f64(weights[f"l{i}.norm1"]), eps)
        h = h + causal_conv(h, f64(weights[f"l{i}.canon1"]))
        y = attention(h, sub(weights, f"l{i}.mix."), layer["mixer"], eps)
        x = x + rms_norm(y, f64(weights[f"l{i}.norm1b"]), eps)
        if layer.get("mlp"):
            h = rms_norm(x, f64(weights[f"l{i}.norm2"]), eps)
            y = routed_ff(h, sub(weights, f"l{i}.mlp."), layer["mlp"])
            x = x + rms_norm(y, f64(weights[f"l{i}.norm2b"]), eps)
        out.append(x.copy())
    return np.stack(out)


def logits(config, weights, tokens):
    """Logits of every position, [n, vocab]."""
    x = layer_streams(config, weights, tokens)[-1]
    return (rms_norm(x, f64(weights["final.norm"]), config["norm"]["eps"]) @ f64(weights["head"]).T) * config["logit_scale"]
