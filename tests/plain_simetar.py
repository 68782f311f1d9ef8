"""A plain, slow Simetar in 64-bit numpy: one function per mechanism, whole sequences only.

Nothing here is shared with the package: no cache, no state, no steps, no kernels.  A sequence is
worked on as a whole, every position from the sequence's first token, so that what the package
does with pages, rings, slots, convolution histories and recorded steps has something
independent to be compared with.

Notation: n tokens, width W; x[t] is row t.  Weights are stored [out, in] and applied as W x.
``w`` of a function: the tensors of that part by their short names.
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


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def layer_norm(x, w, b, eps):
    centred = x - np.mean(x, axis=-1, keepdims=True)
    return centred / np.sqrt(np.mean(centred * centred, axis=-1, keepdims=True) + eps) * w + b


def causal_conv(u, w):
    """u[n, C], w[C, taps]: per channel the weighted sum of the last ``taps`` rows, the row itself
    with the last tap; rows before the sequence's start are zeros."""
    n, taps = u.shape[0], w.shape[1]
    out = np.zeros_like(u)
    for back in range(taps):                     # the row `back` positions ago has tap taps - 1 - back
        if back < n:
            out[back:] += w[:, taps - 1 - back] * u[:n - back]
    return out


def plain_frequencies(dims, base):
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def llama3_frequencies(dims, base, s):
    """Short wavelengths keep their frequency, long ones are slowed down by ``factor``, and between
    the two the share of the plain frequency rises with the number of turns in ``original``
    positions."""
    out = []
    for f in plain_frequencies(dims, base):
        length = 2.0 * math.pi / f
        if length < s["original"] / s["high"]:
            out.append(f)
        elif length > s["original"] / s["low"]:
            out.append(f / s["factor"])
        else:
            share = (s["original"] / length - s["low"]) / (s["high"] - s["low"])
            out.append((1.0 - share) * f / s["factor"] + share * f)
    return out


def yarn_frequencies(dims, base, s):
    """(frequencies, factor on cosine and sine): a straight ramp over the pair's index between the
    indices that make ``fast`` and ``slow`` turns in ``original`` positions."""
    def index_of(turns):
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(index_of(s["fast"])), 0), min(math.ceil(index_of(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain_frequencies(dims, base)):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, dims, freqs, pair_of, magnitude=1.0):
    """Rotary positions on the first ``dims`` entries of the last axis of x[n, heads, d]; row t is
    position t.  ``pair_of(i)`` names the two entries of pair i, whose angle is t freqs[i]; cosine
    and sine are both multiplied by ``magnitude``."""
    y = x.copy()
    t = np.arange(x.shape[0], dtype=np.float64)
    for i in range(dims // 2):
        a, b = pair_of(i)
        c, s = (magnitude * np.cos(t * freqs[i]))[:, None], (magnitude * np.sin(t * freqs[i]))[:, None]
        u, v = x[..., a], x[..., b]
        y[..., a] = u * c - v * s
        y[..., b] = v * c + u * s
    return y


def rotate_neighbours(x, rot):
    """The attention layers' rotation: pairs (2i, 2i + 1)."""
    s = rot.get("scaling")
    freqs = llama3_frequencies(rot["dims"], rot["base"], s) if s else plain_frequencies(rot["dims"], rot["base"])
    return rotate(x, rot["dims"], freqs, lambda i: (2 * i, 2 * i + 1))


def rotate_halves(x, rot):
    """The latent attention layers' rotation: pairs (i, i + dims / 2)."""
    s, half = rot.get("scaling"), rot["dims"] // 2
    freqs, mag = yarn_frequencies(rot["dims"], rot["base"], s) if s else (plain_frequencies(rot["dims"], rot["base"]), 1.0)
    return rotate(x, rot["dims"], freqs, lambda i: (i, i + half), mag)


def softcap(s, cap):
    return cap * np.tanh(s / cap) if cap else s


def weights_beside_one(s):
    """Softmax with a one added to the denominator: e^s / (1 + sum e^s)."""
    top = max(s.max(), 0.0)
    e = np.exp(s - top)
    return e / (np.exp(-top) + e.sum())


def softmax(s):
    e = np.exp(s - s.max())
    return e / e.sum()


def first_visible(t, size):
    return max(0, t - size + 1) if size else 0


def attention(h, w, m, eps):
    """h[n, W] -> [n, W].  Grouped heads whose values are their keys as the convolution leaves
    them; q and k normed as whole rows, then rotated; soft-capped scores in a window, one added
    to the softmax's denominator, a gate per element."""
    n = h.shape[0]
    H, d = m["heads"], m["dim"]
    G = m.get("kv_heads") or H
    q = causal_conv(h @ w["q"].T + w["q.b"], w["q.conv"])
    k = causal_conv(h @ w["k"].T + w["k.b"], w["k.conv"])
    v = k.reshape(n, G, d)
    q = rms_norm(q, w["q.norm"], eps).reshape(n, H, d)
    k = rms_norm(k, w["k.norm"], eps).reshape(n, G, d)
    if m.get("rot"):
        q, k = rotate_neighbours(q, m["rot"]), rotate_neighbours(k, m["rot"])
    size = (m.get("mask") or {}).get("size") or 0
    out = np.zeros((n, H, d))
    for t in range(n):
        lo = first_visible(t, size)
        for a in range(H):
            g = a // (H // G)
            s = softcap(k[lo:t + 1, g] @ q[t, a] * m["scale"], m.get("softcap"))
            out[t, a] = weights_beside_one(s) @ v[lo:t + 1, g]
    return (out.reshape(n, H * d) * sigmoid(h @ w["g"].T)) @ w["o"].T


def latent_rows(h, w, m, eps):
    """What a latent attention layer keeps per position: (the normed latent [n, rank], the rotated
    key part that the heads share [n, rot_dim])."""
    down = h @ w["dkv"].T
    rank = m["kv_rank"]
    shared = down[:, rank:]
    if m.get("rot"):
        shared = rotate_halves(shared[:, None, :], m["rot"])[:, 0]
    return rms_norm(down[:, :rank], w["dkv.norm"], eps), shared


def latent_attention(h, w, m, kept):
    """h[n, W] -> [n, W]; ``kept``: the rows to read (this layer's own or another's)."""
    c, shared = kept
    n = h.shape[0]
    H, d, rd, vd = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = (h @ w["q"].T).reshape(n, H, d + rd)
    qn, qr = q[..., :d], q[..., d:]
    if m.get("rot"):
        qr = rotate_halves(qr, m["rot"])
    k = (c @ w["uk"].T).reshape(n, H, d)
    v = (c @ w["uv"].T).reshape(n, H, vd)
    out = np.zeros((n, H, vd))
    for a in range(H):
        s = (qn[:, a] @ k[:, a].T + qr[:, a] @ shared.T) * m["scale"]
        for t in range(n):
            out[t, a] = softmax(s[t, :t + 1]) @ v[:t + 1, a]
    return (out.reshape(n, H * vd) * sigmoid(h @ w["g"].T)) @ w["o"].T


def dense_ff(h, w):
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def sub(weights, prefix):
    return {k[len(prefix):]: f64(v) for k, v in weights.items() if k.startswith(prefix)}


def layer_streams(config, weights, tokens):
    """The residual stream after every layer, [layers, n, W]."""
    eps = config["norm"]["eps"]
    x = f64(weights["embed"])[np.asarray(tokens, dtype=np.int64)]
    out, kept = [], {}

    def add(x, y, name):
        return x + layer_norm(y, f64(weights[name]), f64(weights[name + ".b"]), eps)
    for i, layer in enumerate(config["layers"]):
        w, m = sub(weights, f"l{i}.mix."), layer["mixer"]
        if layer["type"] == "attention":
            y = attention(x, w, m, eps)
        else:
            if m.get("kv_from") is None:
                kept[i] = latent_rows(x, w, m, eps)
            y = latent_attention(x, w, m, kept[i if m.get("kv_from") is None else m["kv_from"]])
        x = add(x, y, f"l{i}.norm1")
        if layer.get("mlp"):
            x = add(x, dense_ff(x, sub(weights, f"l{i}.mlp.")), f"l{i}.norm2")
        out.append(x.copy())
    return np.stack(out)


def logits(config, weights, tokens):
    """Logits of every position, [n, vocab]."""
    x = layer_streams(config, weights, tokens)[-1]
    return layer_norm(x, f64(weights["final.norm"]), f64(weights["final.norm.b"]),
                      config["norm"]["eps"]) @ f64(weights["head"]).T
