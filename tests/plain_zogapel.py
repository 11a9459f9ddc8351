"""A plain, slow Zogapel in float64 numpy: the oracle of the Zogapel tests.

One function per mechanism, whole sequences, no cache, no batching, nothing shared
with the package.  ``cfg`` is the dictionary of a config.json, ``W`` maps tensor
names to float64 arrays.  X [T, width] is the residual stream of one sequence, t
the position (from 0), rms(x) = sqrt(mean(x^2) + eps), N(x) = x / rms(x) * (1 + w).

    X = E[token] * scale
    layer:   X += N_1b(mix(N_1(X)));   X += N_2b(ff(N_2(X)))
    logits = E N_final(X)
"""

from __future__ import annotations

import math

import numpy as np


def unit_rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.log1p(np.exp(-np.abs(z))) + np.maximum(z, 0.0)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def shifted_norm(x, w, eps):
    """A norm whose weight is stored around zero."""
    return unit_rms(x, eps) * (1.0 + w)


# ----------------------------------------------------------------------------- gated delta rule
def short_conv(x, taps):
    """x [T, C], taps [C, K]: y[t] = sum_j taps[:, K-1-j] x[t-j], zeros before the start."""
    T, K = x.shape[0], taps.shape[1]
    y = np.zeros_like(x)
    for j in range(K):
        y[j:] += taps[:, K - 1 - j] * x[:T - j] if j < T else 0.0
    return y


def unit_vectors(x):
    """x [T, H, D]: every head's vector to length one."""
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


def gated_delta_step(S, g, beta, k, v, q):
    """One token of one head: S [dim, vdim] -> (new S, output).  Decay, then the correction towards v, then the read-out."""
    S = g * S
    S = S + np.outer(k, beta * (v - k @ S))
    return S, q @ S


def gated_delta(h, W, p, c, eps):
    T, H, G, D, DV = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    qkv = {n: silu(short_conv(h @ W[p + n].T, W[p + n + ".conv"])) for n in "qkv"}
    q = unit_vectors(qkv["q"].reshape(T, G, D)) * D ** -0.5
    k = unit_vectors(qkv["k"].reshape(T, G, D))
    v = qkv["v"].reshape(T, H, DV)
    beta = sigmoid(h @ W[p + "b"].T)
    g = np.exp(-np.exp(W[p + "A_log"]) * softplus(h @ W[p + "a"].T + W[p + "dt_bias"]))
    o = np.zeros((T, H, DV))
    for n in range(H):
        S, j = np.zeros((D, DV)), n // (H // G)
        for t in range(T):
            S, o[t, n] = gated_delta_step(S, g[t, n], beta[t, n], k[t, j], v[t, n], q[t, j])
    o = (unit_rms(o, eps) * W[p + "norm"]).reshape(T, H * DV) * silu(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


# ----------------------------------------------------------------------------- attention over keys that are the values
def rotary_frequencies(rot):
    """Angular step of each of the dims/2 pairs, and the factor on cos and sin."""
    dims, base = rot["dims"], float(rot["base"])
    i = np.arange(dims // 2, dtype=np.float64)
    f = base ** (-2.0 * i / dims)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    s, L = float(sc["factor"]), float(sc["original"])
    turn = lambda t: dims * math.log(L / (2.0 * math.pi * t)) / (2.0 * math.log(base))
    lo = max(math.floor(turn(float(sc["fast"]))), 0)
    hi = min(math.ceil(turn(float(sc["slow"]))), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / s * ramp + f * (1.0 - ramp), 0.1 * math.log(s) + 1.0


def rotate(x, rot):
    """x [T, H, D] at positions 0..T-1: element i turns with element i + dims/2; elements from dims on stay."""
    half = rot["dims"] // 2
    f, mag = rotary_frequencies(rot)
    ang = np.arange(x.shape[0], dtype=np.float64)[:, None, None] * f
    cos, sin = np.cos(ang) * mag, np.sin(ang) * mag
    out = x.copy()
    a, b = x[..., :half], x[..., half:2 * half]
    out[..., :half], out[..., half:2 * half] = a * cos - b * sin, b * cos + a * sin
    return out


def window_weights(s, size):
    """Softmax weights of scores s [T, T]: row i sees the columns j with 0 <= i - j < size (size 0: all j <= i)."""
    T = s.shape[0]
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    s = np.where((d >= 0) & ((d < size) if size else True), s, -np.inf)
    w = np.exp(s - s.max(-1, keepdims=True))
    return w / w.sum(-1, keepdims=True)


def tied_attention(h, W, p, c):
    T, H, G, D = h.shape[0], c["heads"], c["kv_heads"], c["dim"]
    q = rotate((h @ W[p + "q"].T).reshape(T, H, D), c["rot"])
    v = (h @ W[p + "k"].T).reshape(T, G, D)
    k = rotate(v, c["rot"])
    size = (c.get("mask") or {}).get("size", 0)
    out = np.zeros((T, H, D))
    for n in range(H):
        j = n // (H // G)
        out[:, n] = window_weights(q[:, n] @ k[:, j].T * float(c["scale"]), size) @ v[:, j]
    out = out.reshape(T, -1) * sigmoid(h @ W[p + "g"].T)
    return out @ W[p + "o"].T


# ----------------------------------------------------------------------------- feed-forwards
def dense(h, W, p):
    return gelu_tanh(h @ W[p + "up"].T) @ W[p + "down"].T


def choose(z, top):
    """(chosen experts, their weights) of one token's logits: the largest ones, softmax over those alone."""
    chosen = np.argsort(-z, kind="stable")[:top]
    w = np.exp(z[chosen] - z[chosen].max())
    return chosen, w / w.sum()


def expert(x, W, p):
    return (silu(x @ W[p + "gate"].T) * (x @ W[p + "up"].T)) @ W[p + "down"].T


def experts(h, W, p, r):
    out = np.zeros_like(h)
    z = h @ W[p + "router"].T + W[p + "router.b"]
    for t in range(h.shape[0]):
        for e, w in zip(*choose(z[t], r["top"])):
            out[t] += w * expert(h[t], W, f"{p}e{e}.")
    return out


# ----------------------------------------------------------------------------- the model
def layer(cfg, W, i, X):
    spec, p, eps = cfg["layers"][i], f"l{i}.", float(cfg["norm"]["eps"])
    h = shifted_norm(X, W[p + "norm1"], eps)
    m = gated_delta(h, W, p + "mix.", spec["mixer"], eps) if spec["type"] == "delta" else tied_attention(h, W, p + "mix.", spec["mixer"])
    X = X + shifted_norm(m, W[p + "norm1b"], eps)
    mlp = spec.get("mlp")
    if not mlp:
        return X
    h = shifted_norm(X, W[p + "norm2"], eps)
    y = experts(h, W, p + "mlp.", mlp["router"]) if mlp["kind"] == "moe" else dense(h, W, p + "mlp.")
    return X + shifted_norm(y, W[p + "norm2b"], eps)


def forward(cfg, W, tokens, streams=None):
    """Logits [T, vocab] of one sequence; ``streams`` (a list) receives the stream after every layer."""
    X = W["embed"][np.asarray(tokens)] * float(cfg["embedding"]["scale"])
    for i in range(len(cfg["layers"])):
        X = layer(cfg, W, i, X)
        if streams is not None:
            streams.append(X.copy())
    return shifted_norm(X, W["final.norm"], float(cfg["norm"]["eps"])) @ W["embed"].T


def greedy(cfg, W, prompt, new_tokens):
    """The prompt's continuation by the largest logit, token by token (each time over the whole sequence)."""
    ids = list(prompt)
    for _ in range(new_tokens):
        ids.append(int(np.argmax(forward(cfg, W, ids)[-1])))
    return ids[len(prompt):]
