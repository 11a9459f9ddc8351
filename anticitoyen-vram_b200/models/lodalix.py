"""The Lodalix design as a plan of parts.

Every layer is a ``parallel`` block over a float32 residual stream: one RMS norm
(its weight stored around zero) in front of a mixer and a feed-forward that run
side by side.  The mixers: ``latent_attention`` with interleaved rotary pairs and a
learned sink; ``latent_attention`` with rotate-half pairs, YaRN scaling and a
sigmoid gate on the heads, some of whose layers read the cache slot of an earlier
one instead of writing their own; ``general_delta``.  The feed-forward is
``swiglu`` with the clamped swish gate and biases, or absent.

What the design fixes is written here as parameters of the parts; what a model
of the design may choose comes from ``LodalixConfig``.
"""

from __future__ import annotations

from ..config.lodalix import MAX_POSITIONS, LatentSpec, LodalixConfig
from ..config.registry import register_architecture
from ..parts.plan import LayerSpec, ModelPlan, PartSpec, ScheduleEntry

SWISH_SLOPE = 1.702         # the gate's g * sigmoid(1.702 g)
NORM_OFFSET = 1.0           # block norms and the final norm multiply by 1 + w
FF_NAMES = {r + b: r + s for r in ("gate", "up", "down") for b, s in (("", ""), (".bias", ".b"))}


def _latent(kind: str, m: LatentSpec, eps: float) -> PartSpec:
    position = PartSpec("rotary", {"dim": m.rot.dims, "theta": m.rot.base, "max_positions": MAX_POSITIONS,
                                   "scaling": m.rot.scaling, "exact": True})
    params = {"num_heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "value_dim": m.vdim, "q_rank": m.q_rank,
              "kv_rank": m.kv_rank, "scale": m.scale, "norm_eps": eps, "position": position, "prefix": "mix."}
    if kind == "latent_attention":
        params.update(sink="sink")
    else:
        params.update(rotate_half=True, gate="g", own_kv=m.kv_from is None)
    return PartSpec("latent_attention", params)


def lodalix_plan(cfg: LodalixConfig) -> ModelPlan:
    norm = PartSpec("rmsnorm", {"eps": cfg.norm_eps, "tensor": "", "offset": NORM_OFFSET})
    layers, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        m = layer.mixer
        if layer.type == "general_delta":
            mixer = PartSpec("general_delta", {"num_heads": m.heads, "dim": m.dim, "norm_eps": cfg.norm_eps, "prefix": "mix."})
        else:
            mixer = _latent(layer.type, m, cfg.norm_eps)
        ff = None
        if layer.mlp is not None:
            ff = PartSpec("swiglu", {"intermediate_size": layer.mlp.ff, "prefix": "mlp.", "bias": True, "names": FF_NAMES,
                                     "activation": "swish_clamped", "limit": layer.mlp.limit, "alpha": SWISH_SLOPE})
        layers.append(LayerSpec(f"l{i}.", "parallel", mixer, ff, norm, norm_prefixes=("norm1", "norm1")))
        source = getattr(m, "kv_from", None)
        # a layer that borrows kept rows reads the slot that their maker writes
        schedule.append(ScheduleEntry(i, i if source is None else source, source is None))
    return ModelPlan(
        architecture=cfg.architecture, hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS,
        layers=tuple(layers), schedule=tuple(schedule), final_norm=norm, embedding_name="embed",
        final_norm_prefix="final.norm", head_name="head", tied_head=False, residual_dtype="float32")


register_architecture("Lodalix", LodalixConfig, lodalix_plan)
