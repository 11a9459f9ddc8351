"""Helpers of the Zogapel tests: small configurations, random weights made to show faults, model folders."""

from __future__ import annotations

import json
import math
import os

import torch
from safetensors.torch import save_file

from vadelix_util import read_folder, row_errors  # noqa: F401  (the tests use them through this module)


def attention(heads, kv_heads, dim, rot, window=0, base=1e4, scaling=None, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale if scale is not None else dim ** -0.5,
         "rot": {"base": base, "dims": rot}}
    if scaling:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if window:
        m["mask"] = {"size": window}
    return "attention", m


def delta(heads, kv_heads, dim, vdim, conv):
    return "delta", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def layer(mixer, mlp):
    return {"type": mixer[0], "mixer": mixer[1], "mlp": mlp}


def model(vocab, width, layers, eps, scale=1.0) -> dict:
    return {"architecture": "Zogapel", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
            "layers": layers}


def config(which: str) -> dict:
    """A: every mechanism at sizes of its own: recurrences with as many and with fewer query heads than value heads, two
       windows (one of a page's size and a bit), scaled and plain rotation of a part of the head, all three feed-forwards.
    B: one head everywhere, whole heads rotated, a window of a single token, one tap, one expert, factors of 1.
    C: sizes that are multiples of nothing (width 100, heads of 10 and 14, recurrence heads of 10 by 7), no window, more taps
       than the recurrence takes tokens at once, every expert chosen, no feed-forward.
    D: sizes of the tensor-core kernels (heads of 64 and 128, 16 to a key head, recurrence heads of 64 by 128 and 128 by 64,
       experts whose steps reach the grouped products)."""
    if which == "A":
        layers = [layer(delta(4, 2, 16, 24, 4), moe(6, 2, 40)),
                  layer(attention(6, 2, 24, 8, 40, 5000.0, (4.0, 64, 16.0, 2.0)), dense(72)),
                  layer(attention(3, 3, 20, 20, 17, 300.0), moe(5, 3, 24)),
                  layer(delta(3, 3, 12, 12, 3), dense(64)),
                  layer(attention(4, 1, 16, 4, 100, 777.0, (2.0, 32, 3.0, 3.0)), None)]
        return model(211, 96, layers, 1e-5, 0.7)
    if which == "B":
        layers = [layer(attention(1, 1, 32, 32, 1, scale=1.0), moe(1, 1, 32)),
                  layer(delta(1, 1, 32, 32, 1), dense(32)),
                  layer(attention(1, 1, 32, 32, 64, 1e4, (1.0, 4096, 32.0, 1.0), scale=1.0), dense(32))]
        return model(300, 64, layers, 1e-6, 1.0)
    if which == "C":
        layers = [layer(attention(3, 3, 10, 6, 0, 50.0), dense(37)),
                  layer(delta(6, 2, 10, 7, 6), moe(5, 5, 22)),
                  layer(attention(4, 2, 14, 2, 33, 900.0, (8.0, 128, 4.0, 1.0)), None),
                  layer(delta(5, 1, 9, 20, 12), dense(44)),
                  layer(delta(2, 1, 40, 4, 2), moe(3, 1, 15))]
        return model(157, 100, layers, 1e-5, 2.5)
    if which == "D":
        layers = [layer(attention(8, 2, 64, 32, 64, 30000.0, (8.0, 128, 16.0, 1.0)), moe(8, 2, 64)),
                  layer(delta(4, 2, 64, 128, 4), dense(160)),
                  layer(attention(16, 1, 128, 24, 100, 1e6), moe(4, 3, 96)),
                  layer(delta(2, 2, 128, 64, 4), None),
                  layer(attention(2, 1, 128, 128, 0, 1e6), dense(128))]
        return model(320, 128, layers, 1e-6, 1.3)
    raise KeyError(which)


def random_weights(cfg: dict, seed: int) -> dict[str, torch.Tensor]:
    """bfloat16 tensors by the design's names.  Matrices give unit-variance outputs for unit-variance inputs; block norms lie
    around zero; decays spread from nothing kept to nearly everything; taps of all places weigh; routers decide clearly and
    their biases matter."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    bf = lambda t: t.to(torch.bfloat16)
    mat = lambda out, inp, gain=1.0: bf(torch.randn(out, inp, generator=g) * gain / math.sqrt(inp))
    vec = lambda n, gain, mean=0.0: bf(mean + gain * torch.randn(n, generator=g))
    t = {"embed": bf(torch.randn(V, W, generator=g)), "final.norm": vec(W, 0.2)}
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        H, G, D, DV = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if lay.get("mlp") else ()):
            t[p + n] = vec(W, 0.2)
        if lay["type"] == "delta":
            K = m["conv"]
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * DV)):
                t[p + "mix." + n] = mat(rows, W, 1.5)
                t[p + f"mix.{n}.conv"] = bf(0.3 + torch.randn(rows, K, generator=g) / math.sqrt(K))
            t[p + "mix.b"], t[p + "mix.a"] = mat(H, W, 1.5), mat(H, W)
            t[p + "mix.A_log"], t[p + "mix.dt_bias"] = vec(H, 1.5, -1.0), vec(H, 1.0, -1.0)
            t[p + "mix.norm"] = vec(DV, 0.2, 1.0)
        else:
            t[p + "mix.q"], t[p + "mix.k"] = mat(H * D, W, 1.5), mat(G * D, W, 1.5)
        t[p + "mix.g"], t[p + "mix.o"] = mat(H * DV, W, 1.5), mat(W, H * DV, 1.5)
        mlp = lay.get("mlp")
        if mlp and mlp["kind"] == "dense":
            t[p + "mlp.up"], t[p + "mlp.down"] = mat(mlp["ff"], W, 1.5), mat(W, mlp["ff"])
        elif mlp:
            E, F = mlp["router"]["experts"], mlp["expert"]["ff"]
            t[p + "mlp.router"], t[p + "mlp.router.b"] = mat(E, W, 12.0), vec(E, 4.0)
            for e in range(E):
                t[f"{p}mlp.e{e}.gate"], t[f"{p}mlp.e{e}.up"] = mat(F, W, 1.5), mat(F, W)
                t[f"{p}mlp.e{e}.down"] = mat(W, F, 1.5)
    return t


def write_model(folder: str, cfg: dict, seed: int, weights: dict | None = None) -> str:
    os.makedirs(folder, exist_ok=True)
    weights = weights if weights is not None else random_weights(cfg, seed)
    with open(os.path.join(folder, "config.json"), "w", encoding="utf-8") as fh:
        json.dump(cfg, fh)
    save_file({n: t.contiguous() for n, t in weights.items()}, os.path.join(folder, "model.safetensors"))
    return folder
