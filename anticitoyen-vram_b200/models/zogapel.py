"""The Zogapel design as a plan of parts.

Every layer is a ``sandwich`` block over a float32 residual stream: an RMS norm (its
weight stored around zero) in front of and behind each of its two parts.  The mixers:
the framework's grouped-query ``attention`` with tied values, a sliding window,
partial rotary positions and an output gate; ``gated_delta``.  The feed-forwards:
``dense`` with the tanh form of gelu; ``moe`` with silu units, a router with a bias,
and the softmax over the chosen logits as weights on the experts' outputs; or none.
The head is the embedding table (without the embedding's scale).

What the design fixes is written here as parameters of the parts; what a model of
the design may choose comes from ``ZogapelConfig``.
"""

from __future__ import annotations

from ..config.registry import register_architecture
from ..config.zogapel import MAX_POSITIONS, DenseSpec, ExpertsSpec, GatedDeltaSpec, TiedAttentionSpec, ZogapelConfig
from ..parts.plan import LayerSpec, ModelPlan, PartSpec, default_schedule

NORM_OFFSET = 1.0           # every norm of the stream multiplies by 1 + w


def _attention(m: TiedAttentionSpec) -> PartSpec:
    position = PartSpec("rotary", {"dim": m.rot.dims, "theta": m.rot.base, "max_positions": MAX_POSITIONS,
                                   "scaling": m.rot.scaling, "exact": True})
    return PartSpec("attention", {
        "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "scale": m.scale, "window": m.window,
        "position": position, "prefix": "mix.", "names": {r: r for r in ("q", "k", "o")}, "bias": False, "tied_values": True,
        "gate": "g"})


def _delta(m: GatedDeltaSpec, eps: float) -> PartSpec:
    return PartSpec("gated_delta", {"num_heads": m.heads, "num_kv_heads": m.kv_heads, "dim": m.dim, "value_dim": m.vdim,
                                    "conv": m.conv, "norm_eps": eps, "prefix": "mix."})


def _feed_forward(f: DenseSpec | ExpertsSpec | None) -> PartSpec | None:
    if f is None:
        return None
    if isinstance(f, DenseSpec):
        return PartSpec("dense", {"intermediate_size": f.ff, "activation": "gelu_tanh", "prefix": "mlp."})
    return PartSpec("moe", {"experts": f.experts, "top": f.top, "expert_ff": f.ff, "expert_unit": "silu", "scoring": "softmax",
                            "renormalize": True, "weight_on": "output", "router_bias": True, "prefix": "mlp."})


def zogapel_plan(cfg: ZogapelConfig) -> ModelPlan:
    norm = PartSpec("rmsnorm", {"eps": cfg.norm_eps, "tensor": "", "offset": NORM_OFFSET})
    layers = []
    for i, layer in enumerate(cfg.layers):
        mixer = _attention(layer.mixer) if isinstance(layer.mixer, TiedAttentionSpec) else _delta(layer.mixer, cfg.norm_eps)
        layers.append(LayerSpec(f"l{i}.", "sandwich", mixer, _feed_forward(layer.mlp), norm, norm_prefixes=("norm1", "norm2"),
                                options={"post_norms": ("norm1b", "norm2b")}))
    return ModelPlan(
        architecture=cfg.architecture, hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS,
        layers=tuple(layers), schedule=default_schedule(len(layers)), final_norm=norm, embedding_name="embed",
        final_norm_prefix="final.norm", head_name="head", tied_head=True, embedding_scale=cfg.embedding_scale,
        residual_dtype="float32")


register_architecture("Zogapel", ZogapelConfig, zogapel_plan)
