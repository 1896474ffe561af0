"""A plain, slow Nekedra in float64 numpy: one function per mechanism, whole sequences only,
loops over tokens and heads.  It shares no code with the engine; the tests hold the engine
against it.

A model is ``(config dict, {tensor name: float64 array})``; ``forward`` returns the logits of
every position and, on request, the residual stream after every layer.
"""

from __future__ import annotations

import math

import numpy as np

UNIT_EPS = 1e-6          # inside the root of the delta mixer's unit vectors


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def scalar_norm(x, g, eps):
    """The model's norm: one learned number for all coordinates."""
    return unit_rms(x, eps) * float(g)


def residual_gate(y, h, w, b):
    """A sublayer's result times a sigmoid of a full product of the sublayer's own input."""
    return y * sigmoid(h @ w.T + b)


# ------------------------------------------------------------------ gated delta rule
def causal_conv(x, taps):
    """x [T, C], taps [C, n]: the last column meets the current token, zeros before the start."""
    t, c = x.shape
    n = taps.shape[1]
    y = np.zeros_like(x)
    for i in range(t):
        for j in range(n):
            src = i - (n - 1) + j
            if src >= 0:
                y[i] += taps[:, j] * x[src]
    return y


def unit_vector(x):
    return x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + UNIT_EPS)


def decay(a, a_log, dt_bias):
    return np.exp(-np.exp(a_log) * softplus(a + dt_bias))


def delta_rule(q, k, v, beta, g):
    """One head: q, k [T, e], v [T, f], beta, g [T] -> [T, f].  The state decays, the key's
    present content is replaced by the step's share of the value, then the query reads."""
    t, e = q.shape
    state = np.zeros((e, v.shape[1]))
    out = np.zeros_like(v)
    for i in range(t):
        state = g[i] * state
        u = beta[i] * (v[i] - state.T @ k[i])
        state = state + np.outer(k[i], u)
        out[i] = state.T @ q[i]
    return out


def delta_mixer(h, w, m, eps):
    t = h.shape[0]
    nh, nk, e, f = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(causal_conv(h @ w["q"].T, w["q.conv"])).reshape(t, nk, e)
    k = silu(causal_conv(h @ w["k"].T, w["k.conv"])).reshape(t, nk, e)
    v = silu(causal_conv(h @ w["v"].T, w["v.conv"])).reshape(t, nh, f)
    q, k = unit_vector(q) * e ** -0.5, unit_vector(k)
    beta = sigmoid(h @ w["b"].T)
    g = decay(h @ w["a"].T, w["A_log"], w["dt_bias"])
    gate = silu(h @ w["g"].T).reshape(t, nh, f)
    o = np.zeros((t, nh, f))
    for head in range(nh):
        kv = head // (nh // nk)
        o[:, head] = delta_rule(q[:, kv], k[:, kv], v[:, head], beta[:, head], g[:, head])
    o = unit_rms(o, eps) * w["norm"] * gate
    return o.reshape(t, nh * f) @ w["o"].T


# ------------------------------------------------------------------ softmax attention
def causal_softmax(q, k, v, scale, sink=None):
    """q [T, H, e], k [T, G, e], v [T, G, f] -> [T, H, f].  ``sink`` [H]: one more term
    exp(sink_h) in the denominator, without key or value."""
    t, n_heads, _ = q.shape
    group = n_heads // k.shape[1]
    out = np.zeros((t, n_heads, v.shape[2]))
    for h in range(n_heads):
        kh, vh = k[:, h // group], v[:, h // group]
        for i in range(t):
            s = (kh[:i + 1] @ q[i, h]) * scale
            top = s.max() if sink is None else max(s.max(), float(sink[h]))
            p = np.exp(s - top)
            den = p.sum() + (0.0 if sink is None else math.exp(float(sink[h]) - top))
            out[i, h] = p @ vh[:i + 1] / den
    return out


def attention_mixer(h, w, m, first_values):
    """Biased projections, no rotation, a sink; ``first_values``: a list that holds the first
    value-mixing layer's values, empty before that layer."""
    t = h.shape[0]
    nh, nk, e, f = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T + w["q.b"]).reshape(t, nh, e)
    k = (h @ w["k"].T + w["k.b"]).reshape(t, nk, e)
    v = (h @ w["v"].T + w["v.b"]).reshape(t, nk, f)
    if m.get("v_mix"):
        if first_values:
            lam = float(w["vmix"])
            v = (1.0 - lam) * v + lam * first_values[0]
        else:
            first_values.append(v)
    o = causal_softmax(q, k, v, m["scale"], sink=w["sink"])
    return o.reshape(t, nh * f) @ w["o"].T


def rotate_pairs(x, dims, base):
    """x [T, ..., n]: entries 2i and 2i + 1 (below ``dims``) turn by position * base^(-2i/dims)."""
    y = x.copy()
    for p in range(x.shape[0]):
        for i in range(dims // 2):
            a = p * base ** (-2.0 * i / dims)
            u, v = x[p, ..., 2 * i], x[p, ..., 2 * i + 1]
            y[p, ..., 2 * i] = u * math.cos(a) - v * math.sin(a)
            y[p, ..., 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return y


def latent_mixer(h, w, m, eps):
    """Keys and values rebuilt from the latent, one rotated key part for all heads, one gate
    a head."""
    t = h.shape[0]
    nh, e, r, f, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    rot = m["rot"]
    q = (h @ w["q"].T).reshape(t, nh, e + r)
    down = h @ w["dkv"].T
    c = unit_rms(down[:, :rank], eps) * w["dkv.norm"]
    k_rot = rotate_pairs(down[:, rank:], rot["dims"], rot["base"])
    q_rot = rotate_pairs(q[:, :, e:], rot["dims"], rot["base"])
    k = (c @ w["uk"].T).reshape(t, nh, e)
    v = (c @ w["uv"].T).reshape(t, nh, f)
    q = np.concatenate([q[:, :, :e], q_rot], axis=2)
    k = np.concatenate([k, np.repeat(k_rot[:, None], nh, axis=1)], axis=2)
    o = causal_softmax(q, k, v, m["scale"]) * sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(t, nh * f) @ w["o"].T


def dense_unit(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


# ------------------------------------------------------------------ the model
def sub(tensors: dict, prefix: str) -> dict:
    return {n[len(prefix) + 1:]: t for n, t in tensors.items() if n.startswith(prefix + ".")}


def forward(config: dict, tensors: dict, tokens, want_layers: bool = False):
    eps = config["norm"]["eps"]
    x = np.stack([tensors["embed"][t] for t in tokens])
    first_values: list = []
    after = []
    for i, layer in enumerate(config["layers"]):
        w, m = sub(tensors, f"l{i}"), layer["mixer"]
        h = scalar_norm(x, w["norm1"], eps)
        mix = sub(w, "mix")
        if layer["type"] == "delta":
            y = delta_mixer(h, mix, m, eps)
        elif layer["type"] == "attention":
            y = attention_mixer(h, mix, m, first_values)
        elif layer["type"] == "latent_attention":
            y = latent_mixer(h, mix, m, eps)
        else:
            raise ValueError(layer["type"])
        x = x + scalar_norm(residual_gate(y, h, w["rg1"], w["rg1.b"]), w["norm1b"], eps)
        if layer.get("mlp") is not None:
            h = scalar_norm(x, w["norm2"], eps)
            y = dense_unit(h, sub(w, "mlp"))
            x = x + scalar_norm(residual_gate(y, h, w["rg2"], w["rg2.b"]), w["norm2b"], eps)
        after.append(x.copy())
    logits = scalar_norm(x, tensors["final.norm"], eps) @ tensors["head"].T
    return (logits, np.stack(after)) if want_layers else logits
