"""A plain, slow Sevazen in float64 numpy: one function per mechanism, whole sequences only,
loops over heads and queries.  It shares no code with the engine; the tests hold the engine
against it.

A model is ``(config dict, {tensor name: float64 array})``; ``forward`` returns the logits of
every position and, on request, the residual stream after every layer.  ``margins``, a list, is
filled with how far every token's last chosen expert lies ahead of the next one.
"""

from __future__ import annotations

import math

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def layer_norm(x, w, b, eps):
    mean = x.mean(axis=-1, keepdims=True)
    var = ((x - mean) ** 2).mean(axis=-1, keepdims=True)
    return (x - mean) / np.sqrt(var + eps) * w + b


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def squared_relu(z):
    return np.maximum(z, 0.0) ** 2


def causal_conv(x, taps):
    """x [T, C], taps [C, n]: the last column meets the current token, zeros before the start."""
    y = np.zeros_like(x)
    n = taps.shape[1]
    for i in range(x.shape[0]):
        for j in range(n):
            src = i - (n - 1) + j
            if src >= 0:
                y[i] += taps[:, j] * x[src]
    return y


# ------------------------------------------------------------------ rotation
def base_frequencies(dims, base):
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def banded_frequency(f, factor, low, high, original):
    """Long wavelengths are stretched, short ones kept, those between mixed."""
    wavelength = 2.0 * math.pi / f
    if wavelength < original / high:
        return f
    if wavelength > original / low:
        return f / factor
    s = (original / wavelength - low) / (high - low)
    return (1.0 - s) * f / factor + s * f


def yarn_frequencies(dims, base, factor, original, fast, slow):
    def dim_of(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(dim_of(fast)), 0)
    hi = min(math.ceil(dim_of(slow)), dims - 1)
    out = []
    for i, f in enumerate(base_frequencies(dims, base)):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out


def frequencies(rot):
    """(frequencies of the pairs, what cosine and sine are multiplied by)"""
    dims, base, s = rot["dims"], rot["base"], rot.get("scaling")
    if s is None:
        return base_frequencies(dims, base), 1.0
    if "fast" in s:
        return (yarn_frequencies(dims, base, s["factor"], s["original"], s["fast"], s["slow"]),
                0.1 * math.log(s["factor"]) + 1.0)
    return [banded_frequency(f, s["factor"], s["low"], s["high"], s["original"])
            for f in base_frequencies(dims, base)], 1.0


def rotate_halves(x, rot):
    """x [T, ..., n]: entry i turns with entry i + dims/2 by position times frequency i."""
    if rot is None:
        return x
    y = x.copy()
    half = rot["dims"] // 2
    freq, amplitude = frequencies(rot)
    for p in range(x.shape[0]):
        for i in range(half):
            c, s = math.cos(p * freq[i]) * amplitude, math.sin(p * freq[i]) * amplitude
            u, v = x[p, ..., i], x[p, ..., i + half]
            y[p, ..., i] = u * c - v * s
            y[p, ..., i + half] = v * c + u * s
    return y


# ------------------------------------------------------------------ attention
def window_start(size):
    return lambda i: max(0, i - size + 1)


def chunk_start(size):
    return lambda i: i // size * size


def visible_softmax(q, k, v, scale, first, sink=None):
    """q [T, H, e], k [T, G, e], v [T, G, f] -> [T, H, f]; position i sees first(i) .. i.
    ``sink`` [H]: one more term exp(sink_h) in the denominator, without key or value."""
    t, n_heads, _ = q.shape
    group = n_heads // k.shape[1]
    out = np.zeros((t, n_heads, v.shape[2]))
    for h in range(n_heads):
        kh, vh = k[:, h // group], v[:, h // group]
        for i in range(t):
            lo = first(i)
            s = (kh[lo:i + 1] @ q[i, h]) * scale
            top = s.max() if sink is None else max(s.max(), float(sink[h]))
            p = np.exp(s - top)
            den = p.sum() + (0.0 if sink is None else math.exp(float(sink[h]) - top))
            out[i, h] = p @ vh[lo:i + 1] / den
    return out


def projected(h, w, name, taps):
    y = h @ w[name].T + w[f"{name}.b"]
    return causal_conv(y, w[f"{name}.conv"]) if taps else y


def window_attention(h, w, m, eps):
    """Biased projections through short convolutions, normed and rotated queries and keys, a
    window, a sink."""
    t = h.shape[0]
    nh, nk, e, f = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    taps, rot = m.get("conv"), m.get("rot")
    q = projected(h, w, "q", taps).reshape(t, nh, e)
    k = projected(h, w, "k", taps).reshape(t, nk, e)
    v = projected(h, w, "v", taps).reshape(t, nk, f)
    q = rotate_halves(unit_rms(q, eps) * w["q.norm"], rot)
    k = rotate_halves(unit_rms(k, eps) * w["k.norm"], rot)
    mask = m.get("mask")
    first = window_start(mask["size"]) if mask else (lambda i: 0)
    o = visible_softmax(q, k, v, m["scale"], first, sink=w["sink"])
    return o.reshape(t, nh * f) @ w["o"].T


def lambda_of(w, diff):
    return math.exp(w["lq1"] @ w["lk1"]) - math.exp(w["lq2"] @ w["lk2"]) + diff


def differential_attention(h, w, m, eps):
    """Two attentions a head over the same values; the second, weighed, is taken from the first;
    normed, scaled and gated."""
    t = h.shape[0]
    nh, nk, e, f = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot, mask = m.get("rot"), m.get("mask")
    q = projected(h, w, "q", None).reshape(t, nh, 2, e)
    k = projected(h, w, "k", None).reshape(t, nk, 2, e)
    v = projected(h, w, "v", None).reshape(t, nk, f)
    q = rotate_halves(unit_rms(q, eps) * w["q.norm"], rot)
    k = rotate_halves(unit_rms(k, eps) * w["k.norm"], rot)
    first = chunk_start(mask["size"]) if mask else (lambda i: 0)
    a1 = visible_softmax(q[:, :, 0], k[:, :, 0], v, m["scale"], first)
    a2 = visible_softmax(q[:, :, 1], k[:, :, 1], v, m["scale"], first)
    o = unit_rms(a1 - lambda_of(w, m["diff"]) * a2, eps) * (1.0 - m["diff"])
    o = o.reshape(t, nh * f) * sigmoid(h @ w["g"].T)
    return o @ w["o"].T


# ------------------------------------------------------------------ feed-forwards
def dense_unit(h, w):
    return squared_relu(h @ w["up"].T) @ w["down"].T


def routed_units(h, w, mlp, margins=None):
    """The experts with the largest logits, weighed by a softmax over those logits; a shared
    expert behind a gate of one number a token."""
    n, top = mlp["router"]["experts"], mlp["router"]["top"]
    z = h @ w["router"].T + w["router.b"]
    y = np.zeros_like(h)
    for t in range(h.shape[0]):
        order = sorted(range(n), key=lambda e: (-z[t, e], e))
        chosen = order[:top]
        if margins is not None and top < n:
            margins.append(z[t, chosen[-1]] - z[t, order[top]])
        p = np.exp(z[t, chosen] - z[t, chosen].max())
        p /= p.sum()
        for weight, e in zip(p, chosen):
            y[t] += weight * dense_unit(h[t], {"up": w[f"e{e}.up"], "down": w[f"e{e}.down"]})
    if mlp.get("shared") is not None:
        y = y + dense_unit(h, {"up": w["shared.up"], "down": w["shared.down"]}) \
            * sigmoid(h @ w["shared.sg"].T)
    return y


# ------------------------------------------------------------------ the model
def sub(tensors: dict, prefix: str) -> dict:
    return {n[len(prefix) + 1:]: t for n, t in tensors.items() if n.startswith(prefix + ".")}


MIXERS = {"attention": window_attention, "attention_2": differential_attention}


def forward(config: dict, tensors: dict, tokens, want_layers: bool = False, margins=None):
    eps = config["norm"]["eps"]
    x = np.stack([tensors["embed"][t] for t in tokens])
    after = []
    for i, layer in enumerate(config["layers"]):
        owner = i
        while config["layers"][owner].get("weights_of") is not None:
            owner = config["layers"][owner]["weights_of"]
        w, mlp = sub(tensors, f"l{owner}"), layer.get("mlp")
        y = MIXERS[layer["type"]](x, sub(w, "mix"), layer["mixer"], eps)
        x = x + layer_norm(y, w["norm1"], w["norm1.b"], eps)
        if mlp is not None:
            y = (dense_unit(x, sub(w, "mlp")) if mlp["kind"] == "dense"
                 else routed_units(x, sub(w, "mlp"), mlp, margins))
            x = x + layer_norm(y, w["norm2"], w["norm2.b"], eps)
        after.append(x.copy())
    logits = layer_norm(x, tensors["final.norm"], tensors["final.norm.b"], eps) @ tensors["embed"].T
    return (logits, np.stack(after)) if want_layers else logits
