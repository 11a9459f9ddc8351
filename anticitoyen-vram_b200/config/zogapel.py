"""Typed configuration of the Zogapel design.

A small decoder-only model over a float32 residual stream.  Every layer puts an RMS
norm (its weight stored around zero) in front of and behind each of its two parts,
x += norm_b(part(norm(x))).  The mixer is one of

  ``attention``  grouped queries under a sliding window; the values are the keys as
                 projected, before rotation; rotary positions on the first part of a
                 head (rotate-half pairs, YaRN scaling); a sigmoid gate on the heads;
  ``delta``      a gated delta rule with a decay and a step size per head, behind a
                 short causal convolution of q, k and v.

The feed-forward is W_down gelu(W_up h), a mixture of gated experts whose router
has a bias, or absent.  The head is the embedding table.  config.json is nested:

    {"architecture": "Zogapel", "vocab": V, "width": W, "embedding": {"scale": s}, "norm": {"eps": e},
     "layers": [{"type": "attention", "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size"},
                 "rot": {"base", "dims", "scaling": {"factor", "original", "fast", "slow"}}},
                 "mlp": null | {"kind": "dense", "ff": F} |
                        {"kind": "moe", "router": {"experts": E, "top": n}, "expert": {"ff": F}}},
                {"type": "delta", "mixer": {"heads", "kv_heads", "dim", "vdim", "conv"}, "mlp": ...}, ...]}

Every size and constant that may differ between models is read from there.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from .base import ConfigError, take_float, take_int
from .redudra import RotarySpec, _section

MAX_POSITIONS = 1 << 17     # rows of the rotary tables; the design itself names no longest sequence


def _heads(m: Mapping[str, Any], where: str) -> tuple[int, int]:
    heads = take_int(m, "heads")
    kv = take_int(m, "kv_heads", heads)
    if heads % kv:
        raise ConfigError(f"{where}heads {heads} is not a multiple of kv_heads {kv}")
    return heads, kv


@dataclass(frozen=True)
class TiedAttentionSpec:
    """Mixer ``attention``."""

    heads: int
    kv_heads: int
    dim: int                    # of a query and of a key, which is its own value
    scale: float
    window: int                 # 0: every earlier key is seen
    rot: RotarySpec

    @classmethod
    def from_dict(cls, m: Mapping[str, Any], where: str) -> "TiedAttentionSpec":
        heads, kv = _heads(m, where)
        dim = take_int(m, "dim", minimum=2)
        if take_int(m, "vdim", dim) != dim:
            raise ConfigError(f"{where}vdim {m['vdim']} differs from dim {dim}: a value is its key")
        mask = _section(m, "mask", where, optional=True)
        return cls(heads, kv, dim, take_float(m, "scale", dim ** -0.5), take_int(mask, "size") if mask is not None else 0,
                   RotarySpec.from_dict(_section(m, "rot", where), where, dim))

    def to_dict(self) -> dict:
        out: dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.dim,
                               "scale": self.scale, "rot": self.rot.to_dict()}
        if self.window:
            out["mask"] = {"size": self.window}
        return out


@dataclass(frozen=True)
class GatedDeltaSpec:
    """Mixer ``delta``."""

    heads: int                  # of values, gates and states
    kv_heads: int               # of queries and keys
    dim: int
    vdim: int
    conv: int                   # taps

    @classmethod
    def from_dict(cls, m: Mapping[str, Any], where: str) -> "GatedDeltaSpec":
        heads, kv = _heads(m, where)
        dim = take_int(m, "dim")
        return cls(heads, kv, dim, take_int(m, "vdim", dim), take_int(m, "conv"))

    def to_dict(self) -> dict:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.conv}


@dataclass(frozen=True)
class DenseSpec:
    ff: int

    def to_dict(self) -> dict:
        return {"kind": "dense", "ff": self.ff}


@dataclass(frozen=True)
class ExpertsSpec:
    experts: int
    top: int
    ff: int                     # of one expert

    def to_dict(self) -> dict:
        return {"kind": "moe", "router": {"experts": self.experts, "top": self.top}, "expert": {"ff": self.ff}}


def _feed_forward(mlp: Any, where: str) -> DenseSpec | ExpertsSpec | None:
    if mlp is None:
        return None
    if not isinstance(mlp, Mapping):
        raise ConfigError(f"{where}'mlp' must be an object or null")
    kind = mlp.get("kind", "dense")
    if kind == "dense":
        return DenseSpec(take_int(mlp, "ff"))
    if kind != "moe":
        raise ConfigError(f"{where}mlp.kind = {kind!r}: the feed-forwards built for this design are: dense, moe")
    router = _section(mlp, "router", where + "mlp.")
    experts, top = take_int(router, "experts"), take_int(router, "top")
    if top > experts:
        raise ConfigError(f"{where}mlp.router.top {top} is more than its {experts} experts")
    return ExpertsSpec(experts, top, take_int(_section(mlp, "expert", where + "mlp."), "ff"))


@dataclass(frozen=True)
class ZogapelLayer:
    type: str                   # "attention" | "delta"
    mixer: TiedAttentionSpec | GatedDeltaSpec
    mlp: DenseSpec | ExpertsSpec | None


@dataclass(frozen=True)
class ZogapelConfig:
    vocab: int
    width: int
    embedding_scale: float
    norm_eps: float
    layers: tuple[ZogapelLayer, ...]

    architecture = "Zogapel"
    MIXERS = {"attention": TiedAttentionSpec, "delta": GatedDeltaSpec}

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @classmethod
    def from_dict(cls, cfg: Mapping[str, Any]) -> "ZogapelConfig":
        raw = cfg.get("layers")
        if not isinstance(raw, (list, tuple)) or not raw:
            raise ConfigError("config key 'layers' must be a non-empty list")
        layers: list[ZogapelLayer] = []
        for i, entry in enumerate(raw):
            where = f"layers[{i}]: "
            if not isinstance(entry, Mapping):
                raise ConfigError(f"{where}must be an object")
            kind = entry.get("type")
            spec = cls.MIXERS.get(kind)
            if spec is None:
                raise ConfigError(f"{where}'type' = {kind!r}: the mixers built for this design are: {', '.join(sorted(cls.MIXERS))}")
            layers.append(ZogapelLayer(kind, spec.from_dict(_section(entry, "mixer", where), where), _feed_forward(entry.get("mlp"), where)))
        embedding = _section(cfg, "embedding", "", optional=True)
        return cls(vocab=take_int(cfg, "vocab"), width=take_int(cfg, "width"),
                   embedding_scale=take_float(embedding, "scale", 1.0) if embedding is not None else 1.0,
                   norm_eps=take_float(_section(cfg, "norm", ""), "eps"), layers=tuple(layers))

    def to_dict(self) -> dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "embedding": {"scale": self.embedding_scale}, "norm": {"eps": self.norm_eps},
                "layers": [{"type": l.type, "mixer": l.mixer.to_dict(), "mlp": l.mlp.to_dict() if l.mlp else None}
                           for l in self.layers]}
