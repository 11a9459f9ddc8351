"""Helpers of the Lodalix tests: small configurations, random weights made to show faults, model folders."""

from __future__ import annotations

import json
import math
import os

import torch
from safetensors.torch import save_file

from vadelix_util import clean, read_folder, row_errors  # noqa: F401  (the tests use them through this module)


def rot(base, dims, scaling=None):
    r = {"base": base, "dims": dims}
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, base, scale=None):
    """The first kind: interleaved pairs, a sink."""
    return "latent_attention", {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                                "scale": scale if scale is not None else (dim + rot_dim) ** -0.5, "rot": rot(base, rot_dim)}


def gated(heads, dim, rot_dim, vdim, q_rank, kv_rank, base, scaling, kv_from=None, scale=None):
    """The second kind: halves, scaled frequencies, a gate; maybe another layer's rows."""
    m = latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, base, scale)[1]
    m["rot"] = rot(base, rot_dim, scaling)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return "latent_attention_2", m


def delta(heads, dim, rank=8):
    return "general_delta", {"heads": heads, "dim": dim, "_rank": rank}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def layer(mixer, mlp):
    return {"type": mixer[0], "mixer": mixer[1], "mlp": mlp}


def model(vocab, width, layers, eps) -> dict:
    return {"architecture": "Lodalix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


def config(which: str) -> dict:
    """A: every mechanism at sizes of its own: a gated layer whose rows a later one reads with other head counts and sizes, a
       recurrence of 3 heads between them, a sink layer, a layer without feed-forward.
    B: one head everywhere, unrotated part, rotated part, values and latents of one size, a scaling factor of 1, a limit
       that no value reaches, one recurrence head, a sharp softmax; the sink layer first.
    C: sizes that are multiples of nothing (width 100, rows of 28 and 35, recurrence heads of 10 and 20 channels), rotated
       parts of 2 elements, two layers read one layer's rows, a scaling whose ramp is a step; a tight limit.
    D: sizes of the tensor-core kernels (width 128, latents of 128 and 256, values of 64 and 128, recurrence heads of 64 and
       128 channels), 20 heads in one layer; rows made by a layer and read at the very end."""
    if which == "A":
        y = (4.0, 64, 16.0, 2.0)
        layers = [layer(gated(3, 16, 8, 24, 40, 48, 5000.0, y), dense(80, 1.2)),
                  layer(delta(3, 16, rank=6), dense(72, 2.0)),
                  layer(latent(4, 12, 12, 20, 36, 32, 300.0), dense(64, 0.9)),
                  layer(gated(5, 8, 8, 16, 24, 48, 5000.0, y, kv_from=0), None),
                  layer(delta(2, 24, rank=5), None)]
        return model(211, 96, layers, 1e-5)
    if which == "B":
        layers = [layer(latent(1, 32, 32, 32, 32, 32, 10000.0, scale=0.9), dense(96, 50.0)),
                  layer(delta(1, 32, rank=1), dense(96, 50.0)),
                  layer(gated(1, 32, 32, 32, 32, 32, 10000.0, (1.0, 4096, 32.0, 1.0), scale=0.9), dense(96, 50.0))]
        return model(300, 64, layers, 1e-6)
    if which == "C":
        y = (2.0, 32, 3.0, 3.0)
        layers = [layer(delta(3, 10, rank=3), dense(60, 0.5)),
                  layer(gated(3, 10, 6, 14, 18, 22, 777.0, y), dense(52, 0.7)),
                  layer(latent(5, 7, 2, 9, 11, 33, 50.0), None),
                  layer(gated(2, 13, 6, 5, 23, 22, 777.0, y, kv_from=1), dense(37, 1.5)),
                  layer(delta(2, 20, rank=7), dense(60, 3.0)),
                  layer(gated(7, 3, 6, 11, 9, 22, 777.0, y, kv_from=1), dense(44, 1.0))]
        return model(157, 100, layers, 1e-5)
    if which == "D":
        y = (8.0, 128, 16.0, 1.0)
        layers = [layer(gated(4, 64, 32, 64, 96, 128, 30000.0, y), dense(160, 1.7)),
                  layer(delta(2, 64, rank=16), dense(192, 1.0)),
                  layer(latent(20, 32, 64, 32, 128, 256, 1e6), dense(128, 1.3)),
                  layer(delta(1, 128, rank=24), dense(160, 2.5)),
                  layer(gated(2, 128, 32, 128, 64, 128, 30000.0, y, kv_from=0), dense(160, 1.1))]
        return model(320, 128, layers, 1e-6)
    raise KeyError(which)


def random_weights(cfg: dict, seed: int) -> dict[str, torch.Tensor]:
    """bfloat16 tensors by the design's names.  Matrices give unit-variance outputs for unit-variance inputs; block norms lie
    around zero, latent norms around one; sinks are of the scores' own size; decays spread over their range (0.55 to 1)
    and removal rates over theirs; biases matter and branches reach their clamps."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    bf = lambda t: t.to(torch.bfloat16)
    mat = lambda out, inp, gain=1.0: bf(torch.randn(out, inp, generator=g) * gain / math.sqrt(inp))
    vec = lambda n, gain, mean=0.0: bf(mean + gain * torch.randn(n, generator=g))
    t = {"embed": bf(torch.randn(V, W, generator=g)), "final.norm": vec(W, 0.2), "head": mat(V, W, 3.0)}
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        t[p + "norm1"] = vec(W, 0.2)
        if lay["type"] == "general_delta":
            H, D, R = m["heads"], m["dim"], m.get("_rank", 8)
            for n in "rkvga":
                t[p + "mix." + n] = mat(H * D, W, 1.2)
            t[p + "mix.a.b"] = vec(H * D, 1.0)
            t[p + "mix.w1"], t[p + "mix.w2"] = mat(R, W, 1.5), mat(H * D, R, 1.5)
            t[p + "mix.w0"] = vec(H * D, 1.5, -1.5)
            t[p + "mix.norm"] = vec(H * D, 0.2, 1.0)
            t[p + "mix.o"] = mat(W, H * D)
        else:
            H, D, R, DV, QR, KR = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"))
            t[p + "mix.dq"], t[p + "mix.dq.norm"] = mat(QR, W), vec(QR, 0.2, 1.0)
            t[p + "mix.uq"] = mat(H * (D + R), QR, 1.5)
            if "kv_from" not in m:
                t[p + "mix.dkv"], t[p + "mix.dkv.norm"] = mat(KR + R, W, 1.3), vec(KR, 0.2, 1.0)
            t[p + "mix.uk"], t[p + "mix.uv"] = mat(H * D, KR, 1.3), mat(H * DV, KR)
            t[p + "mix.o"] = mat(W, H * DV, 1.5)
            if lay["type"] == "latent_attention":
                t[p + "mix.sink"] = vec(H, 1.0, 1.0)
            else:
                t[p + "mix.g"] = mat(H * DV, W, 1.5)
        if lay.get("mlp"):
            F = lay["mlp"]["ff"]
            t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"] = mat(F, W, 1.5), mat(F, W, 1.5), mat(W, F)
            for n, k in (("gate", F), ("up", F), ("down", W)):
                t[f"{p}mlp.{n}.b"] = vec(k, 0.3)
    return t


def write_model(folder: str, cfg: dict, seed: int, weights: dict | None = None) -> str:
    os.makedirs(folder, exist_ok=True)
    weights = weights if weights is not None else random_weights(cfg, seed)
    with open(os.path.join(folder, "config.json"), "w", encoding="utf-8") as fh:
        json.dump(clean(cfg), fh)
    save_file({n: t.contiguous() for n, t in weights.items()}, os.path.join(folder, "model.safetensors"))
    return folder
