"""A plain, slow Lodalix in float64 numpy: the oracle of the Lodalix tests.

One function per mechanism, whole sequences, no cache, no batching, nothing shared
with the package.  ``cfg`` is the dictionary of a config.json, ``W`` maps tensor
names to float64 arrays.  X [T, width] is the residual stream of one sequence, t
the position (from 0), rms(x) = sqrt(mean(x^2) + eps).

    layer:   h = X / rms(X) * (1 + w);   X += mix(h) + ff(h)
    logits = head (X / rms(X) * (1 + w_final))
"""

from __future__ import annotations

import math

import numpy as np


def unit_rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def shifted_norm(x, w, eps):
    """A norm whose weight is stored around zero."""
    return unit_rms(x, eps) * (1.0 + w)


def rotary_frequencies(rot, stretched):
    """Angular step of each of the dims/2 pairs, and the factor on cos and sin (YaRN where ``stretched``)."""
    dims, base = rot["dims"], float(rot["base"])
    i = np.arange(dims // 2, dtype=np.float64)
    f = base ** (-2.0 * i / dims)
    sc = rot.get("scaling") if stretched else None
    if not sc:
        return f, 1.0
    s, L = float(sc["factor"]), float(sc["original"])
    turn = lambda t: dims * math.log(L / (2.0 * math.pi * t)) / (2.0 * math.log(base))
    lo = max(math.floor(turn(float(sc["fast"]))), 0)
    hi = min(math.ceil(turn(float(sc["slow"]))), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / s * ramp + f * (1.0 - ramp), 0.1 * math.log(s) + 1.0


def rotate(x, rot, halves):
    """x [T, ..., n] at positions 0..T-1: pairs of neighbours (2i, 2i+1), or with ``halves`` (i, i + dims/2)."""
    dims = rot["dims"]
    f, mag = rotary_frequencies(rot, halves)
    ang = np.arange(x.shape[0], dtype=np.float64).reshape((-1,) + (1,) * (x.ndim - 1)) * f
    cos, sin = np.cos(ang) * mag, np.sin(ang) * mag
    out = x.copy()
    a = slice(0, dims // 2) if halves else slice(0, dims, 2)
    b = slice(dims // 2, dims) if halves else slice(1, dims, 2)
    out[..., a] = x[..., a] * cos - x[..., b] * sin
    out[..., b] = x[..., b] * cos + x[..., a] * sin
    return out


def kept_rows(h, W, p, c, eps, halves):
    """What a latent layer keeps of every token: the normed latent and the rotated key part."""
    kv = h @ W[p + "dkv"].T
    r = c["kv_rank"]
    return unit_rms(kv[:, :r], eps) * W[p + "dkv.norm"], rotate(kv[:, r:], c["rot"], halves)


def latent_queries(h, W, p, c, eps, halves):
    cq = unit_rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]
    q = (cq @ W[p + "uq"].T).reshape(h.shape[0], c["heads"], c["dim"] + c["rot_dim"])
    return q[..., :c["dim"]], rotate(q[..., c["dim"]:], c["rot"], halves)


def causal_weights(s, sink=None):
    """Softmax weights of the causal scores s [T, T]; ``sink``: a score that takes weight and gives nothing."""
    T = s.shape[0]
    s = np.where(np.tril(np.ones((T, T), dtype=bool)), s, -np.inf)
    top = s.max(-1, keepdims=True)
    if sink is not None:
        top = np.maximum(top, sink)
    w = np.exp(s - top)
    total = w.sum(-1, keepdims=True)
    if sink is not None:
        total = total + np.exp(sink - top)
    return w / total


def latent_attention(h, W, p, c, eps, rows, halves, sinks, gated):
    """Attention over kept rows (latent, rotated key part): per head the keys and values are written out in full."""
    T = h.shape[0]
    latent, key_rot = rows
    q, q_rot = latent_queries(h, W, p, c, eps, halves)
    D, DV = c["dim"], c["vdim"]
    out = np.zeros((T, c["heads"], DV))
    for a in range(c["heads"]):
        k = latent @ W[p + "uk"][a * D:(a + 1) * D].T
        v = latent @ W[p + "uv"][a * DV:(a + 1) * DV].T
        s = (q[:, a] @ k.T + q_rot[:, a] @ key_rot.T) * float(c["scale"])
        out[:, a] = causal_weights(s, float(W[p + "sink"][a]) if sinks else None) @ v
    out = out.reshape(T, -1)
    if gated:
        out = out * sigmoid(h @ W[p + "g"].T)
    return out @ W[p + "o"].T


def delta_step(S, w, a, k, v, r):
    """One token of one head: S [dim, dim] -> (new S, output).  Both terms read the old state."""
    u = k / math.sqrt((k * k).sum() + 1e-6)
    S = w[:, None] * S - np.outer(a * u, u @ S) + np.outer(k, v)
    return S, r @ S


def decays(h, W, p):
    return np.exp(-math.exp(-0.5) * sigmoid(np.tanh(h @ W[p + "w1"].T) @ W[p + "w2"].T + W[p + "w0"]))


def general_delta(h, W, p, c, eps):
    T, H, D = h.shape[0], c["heads"], c["dim"]
    heads = lambda z: z.reshape(T, H, D)
    r, k, v = (heads(h @ W[p + n].T) for n in "rkv")
    w = heads(decays(h, W, p))
    a = heads(sigmoid(h @ W[p + "a"].T + W[p + "a.b"]))
    o = np.zeros((T, H, D))
    for n in range(H):
        S = np.zeros((D, D))
        for t in range(T):
            S, o[t, n] = delta_step(S, w[t, n], a[t, n], k[t, n], v[t, n], r[t, n])
    o = unit_rms(o, eps).reshape(T, H * D) * W[p + "norm"] * sigmoid(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


def clamped_unit(h, W, p, limit):
    g = np.minimum(h @ W[p + "gate"].T + W[p + "gate.b"], limit)
    u = np.clip(h @ W[p + "up"].T + W[p + "up.b"], -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T + W[p + "down.b"]


def layer(cfg, W, i, X, kept):
    """``kept``: {layer: its rows}, filled by the layers that make their own and read by those that borrow them."""
    spec, p, eps = cfg["layers"][i], f"l{i}.", float(cfg["norm"]["eps"])
    h = shifted_norm(X, W[p + "norm1"], eps)
    kind, c = spec["type"], spec["mixer"]
    if kind == "general_delta":
        y = general_delta(h, W, p + "mix.", c, eps)
    else:
        second = kind == "latent_attention_2"
        source = c.get("kv_from")
        if source is None:
            kept[i] = kept_rows(h, W, p + "mix.", c, eps, second)
        y = latent_attention(h, W, p + "mix.", c, eps, kept[i if source is None else source], second, not second, second)
    if spec.get("mlp"):
        y = y + clamped_unit(h, W, p + "mlp.", float(spec["mlp"]["limit"]))
    return X + y


def forward(cfg, W, tokens, streams=None):
    """Logits [T, vocab] of one sequence; ``streams`` (a list) receives the stream after every layer."""
    X = W["embed"][np.asarray(tokens)]
    kept = {}
    for i in range(len(cfg["layers"])):
        X = layer(cfg, W, i, X, kept)
        if streams is not None:
            streams.append(X.copy())
    return shifted_norm(X, W["final.norm"], float(cfg["norm"]["eps"])) @ W["head"].T


def greedy(cfg, W, prompt, new_tokens):
    """The prompt's continuation by the largest logit, token by token (each time over the whole sequence)."""
    ids = list(prompt)
    for _ in range(new_tokens):
        ids.append(int(np.argmax(forward(cfg, W, ids)[-1])))
    return ids[len(prompt):]
