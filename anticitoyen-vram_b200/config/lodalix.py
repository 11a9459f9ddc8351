"""Typed configuration of the Lodalix design.

A small decoder-only model over a float32 residual stream whose layers run their
mixer and their feed-forward side by side: both read the output of the layer's one
norm and both join the stream together.  A layer's mixer is one of three:
``latent_attention`` (queries, keys and values through normed low-rank latents,
interleaved rotary pairs, a learned softmax sink per head), ``latent_attention_2``
(the same latents with rotate-half pairs and YaRN scaling, a sigmoid gate on the
heads; such a layer may read the kept rows of an earlier layer, ``kv_from``,
instead of making its own) or ``general_delta`` (a delta-rule recurrence with a
decay and a removal rate for every key channel).  The feed-forward is a clamped
gated unit with biases, or absent.  config.json is nested:

    {"architecture": "Lodalix", "vocab": V, "width": W, "norm": {"eps": e},
     "layers": [{"type": "latent_attention",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "rot": {"base", "dims"}},
                 "mlp": null | {"kind": "dense", "ff": F, "limit": c}},
                {"type": "latent_attention_2",
                 "mixer": {..., "rot": {"base", "dims", "scaling": {"factor", "original", "fast", "slow"}}, "kv_from": j},
                 "mlp": ...},
                {"type": "general_delta", "mixer": {"heads", "dim"}, "mlp": ...}, ...]}

Every size and constant that may differ between models is read from there (the
inner size of the recurrence's decay is its tensors').
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from .base import ConfigError, take_float, take_int
from .redudra import RotarySpec, _section

MAX_POSITIONS = 1 << 17     # rows of the rotary tables; the design itself names no longest sequence


@dataclass(frozen=True)
class LatentSpec:
    """Mixers ``latent_attention`` and ``latent_attention_2``."""

    heads: int
    dim: int                    # unrotated query/key elements of a head
    rot_dim: int                # rotated ones (the keys' are shared by all heads)
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: RotarySpec
    kv_from: int | None = None  # the layer whose kept rows this one reads; None: it makes its own

    @classmethod
    def from_dict(cls, m: Mapping[str, Any], where: str) -> "LatentSpec":
        dim, rot_dim = take_int(m, "dim"), take_int(m, "rot_dim", minimum=2)
        kv_from = m.get("kv_from")
        if kv_from is not None and (isinstance(kv_from, bool) or not isinstance(kv_from, int) or kv_from < 0):
            raise ConfigError(f"{where}'kv_from' must be the number of an earlier layer, got {kv_from!r}")
        return cls(take_int(m, "heads"), dim, rot_dim, take_int(m, "vdim", dim), take_int(m, "q_rank"), take_int(m, "kv_rank"),
                   take_float(m, "scale", (dim + rot_dim) ** -0.5), RotarySpec.from_dict(_section(m, "rot", where), where, rot_dim),
                   kv_from)

    def to_dict(self) -> dict:
        out: dict[str, Any] = {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim,
                               "q_rank": self.q_rank, "kv_rank": self.kv_rank, "scale": self.scale, "rot": self.rot.to_dict()}
        if self.kv_from is not None:
            out["kv_from"] = self.kv_from
        return out

    def rows_like(self, other: "LatentSpec") -> bool:
        """Whether both keep rows of one meaning (sizes and rotation)."""
        return (self.kv_rank, self.rot_dim, self.rot) == (other.kv_rank, other.rot_dim, other.rot)


@dataclass(frozen=True)
class DeltaSpec:
    """Mixer ``general_delta``."""

    heads: int
    dim: int

    @classmethod
    def from_dict(cls, m: Mapping[str, Any], where: str) -> "DeltaSpec":
        return cls(take_int(m, "heads"), take_int(m, "dim"))

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim}


@dataclass(frozen=True)
class ClampedUnitSpec:
    """Feed-forward ``dense``: its inner size and the clamp of its two branches."""

    ff: int
    limit: float

    @classmethod
    def from_dict(cls, m: Mapping[str, Any], where: str) -> "ClampedUnitSpec":
        kind = m.get("kind", "dense")
        if kind != "dense":
            raise ConfigError(f"{where}mlp.kind = {kind!r}: the design's feed-forward is 'dense'")
        return cls(take_int(m, "ff"), take_float(m, "limit"))

    def to_dict(self) -> dict:
        return {"kind": "dense", "ff": self.ff, "limit": self.limit}


@dataclass(frozen=True)
class LodalixLayer:
    type: str                       # "latent_attention" | "latent_attention_2" | "general_delta"
    mixer: LatentSpec | DeltaSpec
    mlp: ClampedUnitSpec | None


@dataclass(frozen=True)
class LodalixConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[LodalixLayer, ...]

    architecture = "Lodalix"
    MIXERS = {"latent_attention": LatentSpec, "latent_attention_2": LatentSpec, "general_delta": DeltaSpec}

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @classmethod
    def from_dict(cls, cfg: Mapping[str, Any]) -> "LodalixConfig":
        raw = cfg.get("layers")
        if not isinstance(raw, (list, tuple)) or not raw:
            raise ConfigError("config key 'layers' must be a non-empty list")
        layers: list[LodalixLayer] = []
        for i, entry in enumerate(raw):
            where = f"layers[{i}]: "
            if not isinstance(entry, Mapping):
                raise ConfigError(f"{where}must be an object")
            kind = entry.get("type")
            spec = cls.MIXERS.get(kind)
            if spec is None:
                raise ConfigError(f"{where}'type' = {kind!r}: the mixers built for this design are: {', '.join(sorted(cls.MIXERS))}")
            mixer = spec.from_dict(_section(entry, "mixer", where), where)
            if kind == "latent_attention" and mixer.rot.scaling is not None:
                raise ConfigError(f"{where}rot.scaling belongs to 'latent_attention_2'")
            j = getattr(mixer, "kv_from", None)
            if j is not None:
                if kind != "latent_attention_2":
                    raise ConfigError(f"{where}'kv_from' belongs to 'latent_attention_2'")
                if j >= i or layers[j].type != kind or layers[j].mixer.kv_from is not None or not mixer.rows_like(layers[j].mixer):
                    raise ConfigError(f"{where}'kv_from' = {j} must name an earlier layer of the same type that makes its own "
                                      f"rows, with equal kv_rank, rot_dim and rot")
            mlp = entry.get("mlp")
            if mlp is not None and not isinstance(mlp, Mapping):
                raise ConfigError(f"{where}'mlp' must be an object or null")
            layers.append(LodalixLayer(kind, mixer, ClampedUnitSpec.from_dict(mlp, where) if mlp is not None else None))
        return cls(vocab=take_int(cfg, "vocab"), width=take_int(cfg, "width"),
                   norm_eps=take_float(_section(cfg, "norm", ""), "eps"), layers=tuple(layers))

    def to_dict(self) -> dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "layers": [{"type": l.type, "mixer": l.mixer.to_dict(), "mlp": l.mlp.to_dict() if l.mlp else None}
                           for l in self.layers]}
