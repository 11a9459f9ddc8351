"""Zogapel without a GPU: configuration, plan, what every layer keeps, and the oracle's mechanisms by hand."""

from __future__ import annotations

import copy
import math

import numpy as np
import pytest

import plain_zogapel as pz
import zogapel_util as zu
from acvram_b200.cache.manager import PagedNeed, StateNeed
from acvram_b200.config import ConfigError, ZogapelConfig, family_of
from acvram_b200.models import DecoderModel
from acvram_b200.models.zogapel import zogapel_plan
from acvram_b200.parts import PartSpec, build


@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
def test_configuration_round_trip(which):
    raw = zu.config(which)
    cfg = ZogapelConfig.from_dict(raw)
    assert cfg.to_dict() == raw
    assert family_of(raw).config_cls is ZogapelConfig
    assert ZogapelConfig.from_dict(cfg.to_dict()) == cfg


def test_configuration_errors_name_the_key():
    def broken(change, which="A"):
        raw = copy.deepcopy(zu.config(which))
        change(raw)
        with pytest.raises(ConfigError) as e:
            ZogapelConfig.from_dict(raw)
        return str(e.value)

    assert "type" in broken(lambda c: c["layers"][0].update(type="retention"))
    assert "vdim" in broken(lambda c: c["layers"][1]["mixer"].update(vdim=32))
    assert "kv_heads" in broken(lambda c: c["layers"][0]["mixer"].update(kv_heads=3))
    assert "kv_heads" in broken(lambda c: c["layers"][1]["mixer"].update(kv_heads=4))
    assert "rot.dims" in broken(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=26))
    assert "rot.dims" in broken(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7))
    assert "size" in broken(lambda c: c["layers"][1]["mixer"]["mask"].update(size=0))
    assert "conv" in broken(lambda c: c["layers"][0]["mixer"].pop("conv"))
    assert "kind" in broken(lambda c: c["layers"][1]["mlp"].update(kind="glu"))
    assert "top" in broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=7))
    assert "expert" in broken(lambda c: c["layers"][0]["mlp"].pop("expert"))
    assert "eps" in broken(lambda c: c["norm"].pop("eps"))
    assert "scale" in broken(lambda c: c["embedding"].update(scale=0))
    assert "layers" in broken(lambda c: c.update(layers=[]))


def test_plan_and_what_every_layer_keeps():
    cfg = ZogapelConfig.from_dict(zu.config("A"))
    plan = zogapel_plan(cfg)
    assert plan.residual_dtype == "float32" and plan.tied_head and plan.embedding_scale == 0.7
    assert all(l.block == "sandwich" and l.norm.params["offset"] == 1.0 for l in plan.layers)
    assert [l.mixer.kind for l in plan.layers] == ["gated_delta", "attention", "attention", "gated_delta", "attention"]
    assert [l.feed_forward.kind if l.feed_forward else None for l in plan.layers] == ["moe", "dense", "moe", "dense", None]
    assert plan.layers[1].mixer.params["window"] == 40 and plan.layers[1].mixer.params["position"].params["dim"] == 8
    m = DecoderModel(plan)
    assert m.blocks[1].cache_need() == PagedNeed(2, 24, 40)
    assert m.blocks[0].cache_need() == {"state": StateNeed((4, 16, 24), "float32"), "inputs": StateNeed((4, 160), "float32")}
    names = m.tensor_needs()
    assert names["head"].optional and "l1.mix.v" not in names and names["l1.mix.g"].shape == (144, 96)
    assert names["l0.mix.v.conv"].shape == (96, 4) and names["l0.mix.norm"].shape == (24,)
    assert names["l0.mlp.router.b"].shape == (6,) and "l4.norm2" not in names and "l3.norm2b" in names
    assert set(names) - {"head"} == set(zu.random_weights(zu.config("A"), 0))


def test_parts_refuse_what_they_do_not_do():
    rope = PartSpec("rotary", {"dim": 8, "theta": 100.0, "max_positions": 16})
    base = {"num_heads": 2, "num_kv_heads": 1, "head_dim": 8, "position": rope, "tied_values": True}
    for more in ({"value_dim": 16}, {"q_temp": (0.1, 4)}, {"score": {"softcap": 3.0}}):
        with pytest.raises(ValueError):
            build("mixer", PartSpec("attention", {**base, **more}), 16)
    assert build("mixer", PartSpec("attention", {**base, "gate": "g"}), 16).in_size == 16 + 8 + 16
    with pytest.raises(ValueError):
        build("mixer", PartSpec("gated_delta", {"num_heads": 3, "num_kv_heads": 2, "dim": 4, "value_dim": 4, "conv": 2, "norm_eps": 1e-5}), 16)
    with pytest.raises(ValueError):         # silu units are not linear in their input
        build("feed_forward", PartSpec("moe", {"experts": 4, "top": 1, "expert_ff": 8, "expert_unit": "silu", "weight_on": "input"}), 16)
    with pytest.raises(ValueError):
        build("feed_forward", PartSpec("moe", {"experts": 4, "top": 1, "expert_ff": 8}), 16)     # a clamped unit without its limit


def test_convolution_by_hand():
    x, taps = np.array([[1.0], [10.0], [100.0], [1000.0]]), np.array([[3.0, 2.0, 1.0]])      # the last tap is the current token's
    assert np.allclose(pz.short_conv(x, taps)[:, 0], [1.0, 12.0, 123.0, 1230.0])
    assert np.allclose(pz.short_conv(x[:1], taps)[:, 0], [1.0])


def test_delta_step_by_hand():
    S = np.array([[1.0, 2.0], [3.0, 4.0]])
    k, v, q = np.array([0.6, 0.8]), np.array([1.0, -1.0]), np.array([0.0, 2.0])
    got, o = pz.gated_delta_step(S, 0.5, 0.25, k, v, q)
    held = 0.5 * S
    u = 0.25 * (v - k @ held)                               # what stands under the key counts after its decay
    assert np.allclose(got, held + np.outer(k, u)) and np.allclose(o, 2.0 * got[1])      # the read-out sees the write
    full, _ = pz.gated_delta_step(S, 1.0, 1.0, k, v, q)
    assert np.allclose(k @ full, v)                         # a full step replaces what stood under a unit key
    assert np.allclose(pz.unit_vectors(np.array([[[3.0, 4.0]]])), [[[0.6, 0.8]]], atol=1e-6)


def test_values_are_the_unrotated_keys_by_hand():
    """Two tokens, one head of two elements, identity projections: the second token's scores meet rotated keys, its output is
    a mean of the unrotated ones."""
    c = {"heads": 1, "kv_heads": 1, "dim": 2, "scale": 1.0, "rot": {"base": 10.0, "dims": 2}, "mask": {"size": 2}}
    W = {"m.q": np.eye(2), "m.k": np.eye(2), "m.g": np.zeros((2, 2)), "m.o": np.eye(2)}
    h = np.array([[1.0, 0.0], [0.0, 2.0]])
    y = pz.tied_attention(h, W, "m.", c)
    s = [h[1] @ np.array([[math.cos(1.0), math.sin(1.0)], [-math.sin(1.0), math.cos(1.0)]]) @ h[0], 4.0]
    w = np.exp(s) / np.exp(s).sum()
    assert np.allclose(y[1], 0.5 * (w[0] * h[0] + w[1] * h[1])) and np.allclose(y[0], 0.5 * h[0])     # the gate is sigmoid(0)
    c["mask"]["size"] = 1
    assert np.allclose(pz.tied_attention(h, W, "m.", c), 0.5 * h)


def test_window_by_hand():
    w = pz.window_weights(np.zeros((4, 4)), 2)
    assert np.allclose(w, [[1, 0, 0, 0], [0.5, 0.5, 0, 0], [0, 0.5, 0.5, 0], [0, 0, 0.5, 0.5]])
    assert np.allclose(pz.window_weights(np.zeros((4, 4)), 0)[3], 0.25)


def test_scaled_frequencies_by_hand():
    rot = {"base": 10000.0, "dims": 16, "scaling": {"factor": 8.0, "original": 1024, "fast": 32.0, "slow": 1.0}}
    f, mag = pz.rotary_frequencies(rot)
    plain, one = pz.rotary_frequencies({"base": 10000.0, "dims": 16})
    lo, hi = math.floor(16 * math.log(1024 / (2 * math.pi * 32)) / (2 * math.log(1e4))), math.ceil(16 * math.log(1024 / (2 * math.pi)) / (2 * math.log(1e4)))
    assert one == 1.0 and mag == pytest.approx(0.1 * math.log(8.0) + 1.0)
    assert np.allclose(f[:lo + 1], plain[:lo + 1]) and np.allclose(f[hi:], plain[hi:] / 8.0) and f[lo + 1] < plain[lo + 1]


def test_choice_by_hand():
    chosen, w = pz.choose(np.array([0.0, 2.0, -1.0, 2.0 + math.log(3.0)]), 2)
    assert chosen.tolist() == [3, 1] and np.allclose(w, [0.75, 0.25])        # the others' logits take no weight
