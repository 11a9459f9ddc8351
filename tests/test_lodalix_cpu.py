"""Lodalix without a GPU: configuration, plan, what every layer keeps, and the oracle's mechanisms by hand."""

from __future__ import annotations

import math

import numpy as np
import pytest

import lodalix_util as lu
import plain_lodalix as pl
from acvram_b200.cache.manager import PagedNeed, StateNeed
from acvram_b200.config import ConfigError, LodalixConfig, family_of
from acvram_b200.models import DecoderModel
from acvram_b200.models.lodalix import lodalix_plan


@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
def test_configuration_round_trip(which):
    raw = lu.clean(lu.config(which))
    cfg = LodalixConfig.from_dict(raw)
    assert cfg.to_dict() == raw
    assert family_of(raw).config_cls is LodalixConfig
    assert LodalixConfig.from_dict(cfg.to_dict()) == cfg


def test_configuration_errors_name_the_key():
    def broken(change, which="A"):
        raw = lu.clean(lu.config(which))
        change(raw)
        with pytest.raises(ConfigError) as e:
            LodalixConfig.from_dict(raw)
        return str(e.value)

    assert "type" in broken(lambda c: c["layers"][0].update(type="attention"))
    assert "rot.dims" in broken(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10))
    assert "scaling" in broken(lambda c: c["layers"][2]["mixer"]["rot"].update(scaling={"factor": 2.0, "original": 8, "fast": 4.0, "slow": 1.0}))
    assert "limit" in broken(lambda c: c["layers"][0]["mlp"].update(limit=0))
    assert "kind" in broken(lambda c: c["layers"][0]["mlp"].update(kind="moe"))
    assert "eps" in broken(lambda c: c["norm"].pop("eps"))
    assert "kv_rank" in broken(lambda c: c["layers"][0]["mixer"].pop("kv_rank"))
    for j in (3, 4, 2, 1, -1):                              # itself, a later one, another kind, a recurrence, no layer
        assert "kv_from" in broken(lambda c: c["layers"][3]["mixer"].update(kv_from=j))
    assert "kv_from" in broken(lambda c: c["layers"][3]["mixer"].update(kv_rank=40))            # rows of two sizes
    assert "kv_from" in broken(lambda c: c["layers"][3]["mixer"]["rot"].update(base=77.0))      # two rotations
    assert "kv_from" in broken(lambda c: c["layers"][5]["mixer"].update(kv_from=3), "C")        # a borrower is no source


def test_plan_and_what_every_layer_keeps():
    cfg = LodalixConfig.from_dict(lu.clean(lu.config("A")))
    plan = lodalix_plan(cfg)
    assert plan.residual_dtype == "float32" and all(l.block == "parallel" for l in plan.layers)
    assert [(e.layer, e.cache, e.writes) for e in plan.schedule] == [(0, 0, True), (1, 1, True), (2, 2, True), (3, 0, False), (4, 4, True)]
    assert [l.mixer.kind for l in plan.layers] == ["latent_attention", "general_delta", "latent_attention", "latent_attention", "general_delta"]
    assert plan.layers[2].mixer.params["sink"] == "sink" and "gate" not in plan.layers[2].mixer.params
    assert plan.layers[3].mixer.params["gate"] == "g" and plan.layers[3].mixer.params["own_kv"] is False
    assert plan.layers[3].feed_forward is None and plan.layers[0].feed_forward.params["limit"] == 1.2
    assert plan.final_norm.params["offset"] == 1.0
    model = DecoderModel(plan)
    rows = PagedNeed(1, 56, 0, 48, 0, 0, True)
    assert model.blocks[0].cache_need() == rows == model.blocks[3].cache_need()
    assert model.blocks[1].cache_need() == StateNeed((3, 16, 16), "float32")
    cplan = model.cache_plan()
    # the borrower has no slot of its own: slot 3 keeps nothing
    assert cplan.needs[0] == rows and cplan.needs[3] is None and cplan.needs[4] == StateNeed((2, 24, 24), "float32")
    names = model.tensor_needs()
    assert "l3.mix.dkv" not in names and "l3.mix.uk" in names and names["l3.mix.g"].shape == (80, 96)
    assert "l2.mix.sink" in names and "l0.mix.sink" not in names and "l3.norm1" in names and "l0.norm2" not in names
    assert names["l0.mlp.down.b"].shape == (96,) and not names["l0.mlp.down.b"].optional
    assert set(names) == set(lu.random_weights(lu.config("A"), 0))


def test_blocks_and_contexts_of_a_step():
    from acvram_b200.kernels import ops
    arrays, values = ops.delta_work([1, 17, 8, 9])
    assert values == {"n_items": 7}
    assert arrays["seg_seq"].tolist() == [0, 1, 1, 1, 2, 3, 3] and arrays["seg_idx"].tolist() == [0, 0, 1, 2, 0, 0, 1]
    assert arrays["first_block"].tolist() == [0, 1, 4, 5]
    # portions that bring few queries for a long context leave it as it is; one-token requests never count
    assert ops.latent_context_work([1, 1], [500, 900])[1]["n_pages"] == 0
    assert ops.latent_context_work([2, 1], [500, 900])[1]["n_pages"] == 0
    assert ops.latent_context_work([2, 100], [100000, 100000])[1]["n_pages"] == 0        # more rows than a step writes out
    arrays, values = ops.latent_context_work([1, 100, 128], [500, 129, 128])
    assert values == {"n_pages": 3, "width": 2} and arrays["order"].tolist() == [0]
    assert arrays["page_seq"].tolist() == [1, 1, 2] and arrays["page_idx"].tolist() == [0, 1, 0]
    assert arrays["table"].reshape(3, 2).tolist() == [[-1, -1], [0, 1], [2, -1]]


def test_rotation_by_hand():
    x = np.arange(8.0).reshape(2, 4)                        # positions 0 and 1, one vector each
    r = lu.rot(100.0, 4)
    near, halves = pl.rotate(x, r, False), pl.rotate(x, r, True)
    assert np.allclose(near[0], x[0]) and np.allclose(halves[0], x[0])
    c, s, c2, s2 = math.cos(1.0), math.sin(1.0), math.cos(0.1), math.sin(0.1)
    assert np.allclose(near[1], [4 * c - 5 * s, 5 * c + 4 * s, 6 * c2 - 7 * s2, 7 * c2 + 6 * s2])
    assert np.allclose(halves[1], [4 * c - 6 * s, 5 * c2 - 7 * s2, 6 * c + 4 * s, 7 * c2 + 5 * s2])


def test_scaled_frequencies_by_hand():
    # turns(32) and turns(1) of 16 dims at base 10000 and 1024 positions: pairs below the first keep their speed, pairs
    # above the second turn `factor` times slower
    f, mag = pl.rotary_frequencies(lu.rot(10000.0, 16, (8.0, 1024, 32.0, 1.0)), True)
    plain, one = pl.rotary_frequencies(lu.rot(10000.0, 16), True)
    lo, hi = math.floor(16 * math.log(1024 / (2 * math.pi * 32)) / (2 * math.log(1e4))), math.ceil(16 * math.log(1024 / (2 * math.pi)) / (2 * math.log(1e4)))
    assert one == 1.0 and mag == pytest.approx(0.1 * math.log(8.0) + 1.0)
    assert np.allclose(f[:lo + 1], plain[:lo + 1]) and np.allclose(f[hi:], plain[hi:] / 8.0) and f[lo + 1] < plain[lo + 1]


def test_sink_and_mask_by_hand():
    s = np.array([[0.0, 9.0], [0.0, 0.0]])
    assert np.allclose(pl.causal_weights(s), [[1.0, 0.0], [0.5, 0.5]])
    assert np.allclose(pl.causal_weights(s, 0.0), [[0.5, 0.0], [1 / 3, 1 / 3]])       # the sink is a further key of score 0
    assert np.allclose(pl.causal_weights(s, math.log(2.0)), [[1 / 3, 0.0], [0.25, 0.25]])


def test_delta_step_by_hand():
    S = np.array([[1.0, 2.0], [3.0, 4.0]])
    k, v, r = np.array([3.0, 4.0]), np.array([1.0, -1.0]), np.array([1.0, 1.0])
    w, a = np.array([0.5, 1.0]), np.array([1.0, 0.5])
    u = k / 5.0                                             # (the 1e-6 beside 25 is below the tolerance)
    seen = u @ S                                            # what both terms read: the old state
    want = np.diag(w) @ S - np.outer(a * u, seen) + np.outer(k, v)
    got, o = pl.delta_step(S, w, a, k, v, r)
    assert np.allclose(got, want, atol=1e-6) and np.allclose(o, want.sum(0), atol=1e-6)
    # no decay and full removal: what stood under u is gone
    S2, _ = pl.delta_step(S, np.ones(2), np.ones(2), k, np.zeros(2), r)
    assert np.allclose(u @ S2, 0.0, atol=1e-5)


def test_clamps_by_hand():
    W = {"m.gate": np.eye(2), "m.gate.b": np.array([0.0, 5.0]), "m.up": np.eye(2), "m.up.b": np.array([-9.0, 0.25]),
         "m.down": np.eye(2), "m.down.b": np.array([10.0, 0.0])}
    y = pl.clamped_unit(np.array([[-3.0, 0.5]]), W, "m.", 1.5)
    # a gate has no lower clamp; an up branch has both
    assert np.allclose(y, [[-3.0 * pl.sigmoid(-5.106) * (-1.5 + 1.0) + 10.0, 1.5 * pl.sigmoid(2.553) * 1.75]])
