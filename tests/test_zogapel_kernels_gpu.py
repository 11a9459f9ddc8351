"""The kernels of the Zogapel parts one by one, each against the oracle's function of the same mechanism on the same
(bfloat16-rounded) inputs: a request's tokens cut into steps of several sizes (down to one and two tokens) against the
whole sequence, states and kept inputs in slots that are not the requests' indices, decays from everything to nothing, keys
planted on both sides of a window's edge, output gates in every attention kernel, routers decided by their bias."""

from __future__ import annotations

import math

import numpy as np
import pytest
import torch

import plain_zogapel as pz
from test_nizedra_kernels_gpu import paged_case
from test_vadelix_kernels_gpu import DEV, DT, batches, bf, close, dev, i32, step_arrays

pytestmark = pytest.mark.gpu

CUTS = ([1] * 9, [2, 2, 2, 2, 1], [9], [3, 1, 5], [1, 8], [7, 2], [4, 5])


# --------------------------------------------------------------------------- the gated delta rule
def delta_weights(rng, width, H, G, D, DV, K, decay_at=-1.0):
    W = {}
    for n, rows in (("q", G * D), ("k", G * D), ("v", H * DV)):
        W["x." + n] = bf(1.5 * rng.standard_normal((rows, width)) / math.sqrt(width))
        W[f"x.{n}.conv"] = bf(0.3 + rng.standard_normal((rows, K)) / math.sqrt(K))
    W.update({"x.b": bf(1.5 * rng.standard_normal((H, width)) / math.sqrt(width)), "x.a": bf(rng.standard_normal((H, width)) / math.sqrt(width)),
              "x.A_log": bf(decay_at + 1.5 * rng.standard_normal(H)), "x.dt_bias": bf(rng.standard_normal(H) - 1.0),
              "x.norm": bf(1.0 + 0.2 * rng.standard_normal(DV)), "x.g": bf(1.5 * rng.standard_normal((H * DV, width)) / math.sqrt(width)),
              "x.o": np.eye(H * DV)})
    return W


class DeltaCase:
    """The kernels' arguments for weights of ``delta_weights``."""

    def __init__(self, W, H, G, D, DV, K, slots):
        self.W, self.sizes, self.K = W, (H, G, D, DV), K
        self.taps_t = dev(np.concatenate([W[f"x.{n}.conv"] for n in "qkv"]).T.copy())
        self.rate, self.shift = dev(np.exp(W["x.A_log"])), dev(W["x.dt_bias"])
        self.weight = dev(np.tile(W["x.norm"], H))
        self.state = torch.zeros((slots, H, D, DV), device=DEV)
        self.ring = torch.zeros((slots, K, 2 * G * D + H * DV), device=DEV)

    def zero(self):
        self.state.zero_()
        self.ring.zero_()

    def run(self, h, step, slots_of, out):
        """The tokens h of a step [(request, first token, count)], the heads into ``out``."""
        from acvram_b200.kernels import ops
        H, G, D, DV = self.sizes
        W = self.W
        proj = dev(np.concatenate([h @ W["x." + n].T for n in ("q", "k", "v", "g", "b", "a")] + [np.zeros((len(h), 3))], axis=1))
        cu, _ = step_arrays(step)
        q_lens = [c for _, _, c in step]
        arrays, values = ops.delta_work(q_lens)
        positions = i32([a + j for _, a, c in step for j in range(c)])
        slots = i32([slots_of[r] for r, _, _ in step])
        ops.gated_delta(proj, self.taps_t, self.rate, self.shift, self.weight, 1e-5, self.ring, slots, self.state, slots, positions,
                        cu, len(step), max(q_lens), out, H, G, D, DV, {**{k: i32(v) for k, v in arrays.items()}, **values})


SHAPES = [(2, 1, 8, 8, 4), (1, 1, 4, 4, 1), (3, 3, 10, 7, 6), (4, 2, 16, 24, 2), (6, 2, 20, 12, 3), (2, 2, 32, 64, 4), (5, 1, 48, 20, 12),
          (4, 2, 64, 128, 4), (2, 1, 100, 36, 9), (4, 2, 128, 128, 4), (9, 1, 128, 16, 5), (1, 1, 200, 256, 4), (2, 1, 300, 8, 3)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D,DV,K", SHAPES)
def test_gated_delta_over_steps(H, G, D, DV, K, dtype):
    """Three requests side by side, cut differently, in slots 4, 0 and 2: portions through blocks, recurrence and gate, steps
    of single tokens through the one-launch kernel where the head allows it.  The convolution reaches over every cut."""
    rng = np.random.default_rng(H * 1000 + D)
    width, I = 40, H * DV
    lengths, slots_of = (9, 21, 14), (4, 0, 2)
    W = delta_weights(rng, width, H, G, D, DV, K)
    hs = [bf(rng.standard_normal((n, width))) for n in lengths]
    case = DeltaCase(W, H, G, D, DV, K, 5)
    got = [np.zeros((n, I)) for n in lengths]
    wants = [pz.gated_delta(h, W, "x.", {"heads": H, "kv_heads": G, "dim": D, "vdim": DV}, 1e-5) for h in hs]
    for cuts in ((CUTS[0], CUTS[0], CUTS[0]), (CUTS[1], CUTS[2], CUTS[5]), (CUTS[3], CUTS[4], CUTS[6]), ([9], [21], [14])):
        case.zero()
        for step in batches(lengths, cuts):
            h = np.concatenate([hs[r][a:a + c] for r, a, c in step])
            wide = torch.full((len(h), I + 5), 7.0, device=DEV, dtype=DT[dtype])       # the heads land in columns of wider rows
            case.run(h, step, slots_of, wide[:, :I])
            assert bool((wide[:, I:] == 7.0).all())
            at = 0
            for r, a0, c in step:
                got[r][a0:a0 + c] = wide[at:at + c, :I].float().cpu().numpy()
                at += c
        for r in range(3):
            close(got[r], wants[r], 1e-4 if dtype == "float32" else 1e-2, f"request {r}, cuts {cuts[r]}")
        assert float(case.state[[1, 3]].abs().max()) == 0.0 == float(case.ring[[1, 3]].abs().max())      # slots of nobody


@pytest.mark.parametrize("D,DV", [(12, 8), (64, 64), (128, 128)])
def test_a_long_portion_equals_token_by_token(D, DV):
    """300 tokens of one request as one portion (many blocks of eight tokens), one by one and cut around a single token;
    decays close to 1 and small steps, so that the first tokens still weigh at the end."""
    rng = np.random.default_rng(D)
    n, H, G, K, width = 300, 2, 1, 4, 32
    W = delta_weights(rng, width, H, G, D, DV, K, decay_at=-9.0)
    W["x.b"], W["x.dt_bias"] = np.zeros((H, width)), W["x.dt_bias"] - 2.0
    # every key alike: what a token writes, half of it stays and the next correction meets it
    h = bf(rng.standard_normal((n, width)))
    c = {"heads": H, "kv_heads": G, "dim": D, "vdim": DV}
    want = pz.gated_delta(h, W, "x.", c, 1e-5)
    if D > 12:
        short = pz.gated_delta(h[40:], W, "x.", c, 1e-5)
        assert float(np.abs(short[-1] - want[-1]).max()) > 1e-3 * float(np.abs(want[-1]).max()), "the first tokens do not matter here"
    case = DeltaCase(W, H, G, D, DV, K, 2)
    for cuts in ([n], [1] * n, [130, 1, 169], [31, 33, 32, 8, 196]):
        case.zero()
        got = torch.empty((n, H * DV), device=DEV)
        at = 0
        for q in cuts:
            case.run(h[at:at + q], [(0, at, q)], (1,), got[at:at + q])
            at += q
        close(got, want, 2e-4, f"cuts {cuts[:3]}")


@pytest.mark.parametrize("rate", [-30.0, 6.0])
def test_decays_at_both_ends(rate):
    """Decays that are 1 to the last place and decays that are 0: products of a block's decays neither overflow nor
    are divided by."""
    rng = np.random.default_rng(3)
    n, H, G, D, DV, K, width = 45, 4, 2, 32, 16, 4, 24
    W = delta_weights(rng, width, H, G, D, DV, K)
    W["x.A_log"] = np.array([rate, rate, 0.0, rate])
    W["x.a"] = 4.0 * W["x.a"]
    h = bf(rng.standard_normal((n, width)))
    want = pz.gated_delta(h, W, "x.", {"heads": H, "kv_heads": G, "dim": D, "vdim": DV}, 1e-5)
    case = DeltaCase(W, H, G, D, DV, K, 1)
    for cuts in ([n], [1] * n, [20, 2, 23]):
        case.zero()
        got = torch.empty((n, H * DV), device=DEV)
        at = 0
        for q in cuts:
            case.run(h[at:at + q], [(0, at, q)], (0,), got[at:at + q])
            at += q
        assert bool(torch.isfinite(got).all())
        close(got, want, 2e-4, f"cuts {cuts[:3]}")


@pytest.mark.parametrize("K", [2, 4, 9, 12])
def test_the_oldest_tap_reaches_over_every_cut(K):
    """Taps that pass the oldest input alone: a value comes out K - 1 tokens late, whatever the cut, and nothing before."""
    rng = np.random.default_rng(K)
    n, H, G, D, DV, width = 30, 2, 1, 8, 12, 16
    W = delta_weights(rng, width, H, G, D, DV, K)
    for name in "qkv":
        W[f"x.{name}.conv"] = np.zeros_like(W[f"x.{name}.conv"])
        W[f"x.{name}.conv"][:, 0] = 1.0
    h = bf(rng.standard_normal((n, width)))
    want = pz.gated_delta(h, W, "x.", {"heads": H, "kv_heads": G, "dim": D, "vdim": DV}, 1e-5)
    assert float(np.abs(want[:K - 1]).max()) == 0.0
    case = DeltaCase(W, H, G, D, DV, K, 1)
    for cuts in ([n], [1] * n, [2] * 15, [5, 1, 24], [13, 2, 1, 1, 13]):
        case.zero()
        got = torch.full((n, H * DV), 7.0, device=DEV)
        at = 0
        for q in cuts:
            case.run(h[at:at + q], [(0, at, q)], (0,), got[at:at + q])
            at += q
        close(got, want, 1e-4, f"cuts {cuts[:3]}")
        assert float(got[:K - 1].abs().max()) == 0.0


# --------------------------------------------------------------------------- keys that are values, the rotated part of a head
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("NH,NKV,D,R", [(4, 2, 64, 32), (3, 1, 128, 24), (2, 2, 128, 128), (2, 1, 128, 20), (5, 5, 10, 6), (1, 1, 32, 2),
                                        (2, 1, 96, 8), (4, 1, 256, 64)])
def test_keys_and_values_into_their_pages(NH, NKV, D, R, dtype):
    """Queries turned in place; keys turned and values as projected, both from the same columns; the gate's columns behind
    them and the elements behind the rotated part stay as they are."""
    from acvram_b200.kernels import ops
    from acvram_b200.parts.base import Runtime
    from acvram_b200.parts.position import Rotary
    rng = np.random.default_rng(NH + R)
    T, page, t = 21, 8, DT[dtype]
    rot = {"base": 700.0, "dims": R, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}}
    part = Rotary(1, R, 700.0, 64, scaling=(4.0, 64, 8.0, 1.0), exact=True)
    part.load({}, Runtime(torch.device(DEV), t))
    x = bf(rng.standard_normal((T, NH + NKV, D)))
    tail = torch.full((T, 8), 5.0, device=DEV, dtype=t)
    qkv = torch.cat([dev(x.reshape(T, -1), t), tail], dim=1).contiguous()
    table = torch.tensor([[-1, -1, -1], [4, 1, 2]], dtype=torch.int32, device=DEV)
    kp, vp = (torch.full((6, NKV, page, D), 9.0, device=DEV, dtype=t) for _ in range(2))
    ops.qk_norm_rope_append(qkv, NH, NKV, D, None, None, 0.0, part.rotary_table(), i32(range(T)), i32([0] * T), table, kp, vp,
                            table_rows=i32([1]), tied=True)
    tol = 1e-5 if dtype == "float32" else 1e-2
    close(qkv[:, :NH * D].view(T, NH, D), pz.rotate(x[:, :NH], rot), tol, "queries")
    assert bool((qkv[:, (NH + NKV) * D:] == 5.0).all())
    order = torch.tensor([4, 1, 2])
    rows = lambda p: p[order].transpose(1, 2).reshape(3 * page, NKV, D)
    close(rows(kp)[:T], pz.rotate(x[:, NH:], rot), tol, "keys")
    assert np.array_equal(rows(vp)[:T].float().cpu().numpy(), x[:, NH:].astype(np.float32))
    for p in (kp, vp):
        assert bool((rows(p)[T:] == 9.0).all()) and bool((p[[0, 3, 5]] == 9.0).all())


# --------------------------------------------------------------------------- output gates
GATE_CASES = [
    # NH NKV  D  page  lens              q_lens        window
    (4, 2, 64, 16, [200, 150, 97], [130, 1, 2], 0),         # tcgen05 portions, split-KV decode, two tokens
    (8, 1, 128, 64, [300, 290], [200, 1], 100),             # under a window
    (3, 1, 40, 16, [70, 33], [40, 1], 30),                  # the generic kernel
    (16, 1, 128, 16, [900, 40, 1300], [1, 1, 1], 0),        # shares of a request's keys merged inside clusters
    (8, 8, 64, 64, [6000, 5000], [1, 1], 0),                # and merged by the last arriver
    (2, 1, 128, 8, [131, 9], [1, 1], 64),                   # small pages
    (5, 5, 64, 128, [140, 500], [139, 3], 0),
    (40, 2, 64, 16, [90, 61, 17], [30, 1, 1], 50),          # more heads to a key head than the tensor-core kernels take
    (4, 2, 256, 16, [50, 33], [20, 1], 20),
]


@pytest.mark.parametrize("case", GATE_CASES, ids=lambda c: f"h{c[0]}d{c[2]}w{c[6]}")
def test_output_gates(case):
    """Every attention kernel with gates far below, around and far above zero, against dense sums in float64; one key planted
    at the window's last place and one a place further back."""
    from acvram_b200.kernels import ops
    NH, NKV, D, page, lens, q_lens, window = case
    ctx, work, table, k, v, T = paged_case(NKV, D, D, page, lens, q_lens, 17 + NH, torch.bfloat16)
    g = torch.Generator().manual_seed(NH + D)
    q = torch.randn(T, NH * D, generator=g)
    q = (q / q.pow(2).mean(-1, keepdim=True).sqrt()).to(torch.bfloat16).to(DEV)
    n, last = lens[0], q_lens[0] - 1
    for place in ([n - window, n - window - 1] if window else [0, page - 1]):
        if 0 <= place < n - 1:
            k[table[0, place // page].item(), :, place % page] = q[last, :D]
    row = torch.randn(T, NH * D + 64, generator=g) * 3.0
    row[:, ::7], row[:, 3::11] = -40.0, 40.0
    row = row.to(torch.bfloat16).to(DEV)
    gate = row[:, 64:]
    scale = D ** -0.5 * 2.0
    want = np.zeros((T, NH, D))
    t0 = 0
    for b, (n, ql) in enumerate(zip(lens, q_lens)):
        js = torch.arange(n)
        pg = table[b].long().cpu()[js // page]
        kk, vv = k.cpu().double()[pg, :, js % page].numpy(), v.cpu().double()[pg, :, js % page].numpy()
        qq = q[t0:t0 + ql].cpu().double().view(ql, NH, D).numpy()
        for h in range(NH):
            j = h // (NH // NKV)
            for i in range(ql):
                p = n - ql + i
                lo = max(0, p - window + 1) if window else 0
                s = qq[i, h] @ kk[lo:p + 1, j].T * scale
                w = np.exp(s - s.max())
                want[t0 + i, h] = (w / w.sum()) @ vv[lo:p + 1, j]
        t0 += ql
    want = want.reshape(T, -1) * pz.sigmoid(gate.cpu().double().numpy())
    top = float(np.abs(want).max())
    out = torch.full((T, NH * D), 7.0, device=DEV, dtype=torch.bfloat16)
    ops.attention(q, out, k, v, ctx, table, NH, NKV, D, scale, window, work=work, gate=gate)
    assert float(np.abs(out.cpu().double().numpy() - want).max()) < 2e-2 * top
    out32 = torch.full((T, NH * D), 7.0, device=DEV)
    ops.attention(q.float(), out32, k.float(), v.float(), ctx, table, NH, NKV, D, scale, window, work=work, gate=gate.float())
    assert float(np.abs(out32.cpu().double().numpy() - want).max()) < 2e-4 * top
    # several splits of every request's keys, whatever the dispatch would choose
    if work["n_dec"] == T and D in (64, 128):
        for splits, cluster in ((1, True), (3, True), (4, False)):
            out.fill_(7.0)
            ops.attention_decode(q, out, k, v, work["dec_tokens"], work["dec_seqs"], T, ctx.kv_len, table, NH, NKV, D, scale, window,
                                 splits, max(lens), cluster_merge=cluster, gate=gate)
            assert float(np.abs(out.cpu().double().numpy() - want).max()) < 2e-2 * top, f"{splits} splits"


# --------------------------------------------------------------------------- experts, dense unit
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,H,F,E,top", [(1, 64, 48, 4, 2), (9, 100, 22, 5, 5), (40, 96, 40, 6, 1), (70, 52, 15, 3, 2), (600, 128, 96, 8, 2),
                                         (400, 128, 64, 4, 3), (5, 64, 64, 1, 1)])
def test_silu_experts_behind_a_biased_router(T, H, F, E, top, dtype):
    """The part as a whole against the oracle's mixture, through the CUDA-core, the mma.sync and the grouped tcgen05 products."""
    from acvram_b200.parts.base import Runtime
    from acvram_b200.parts.feed_forward import RoutedExperts
    rng = np.random.default_rng(T + H)
    W = {"m.router": bf(4.0 * rng.standard_normal((E, H)) / math.sqrt(H)), "m.router.b": bf(2.0 * rng.standard_normal(E))}
    for e in range(E):
        for n, shape in (("gate", (F, H)), ("up", (F, H)), ("down", (H, F))):
            W[f"m.e{e}.{n}"] = bf(1.5 * rng.standard_normal(shape) / math.sqrt(shape[1]))
    part = RoutedExperts(H, E, top, F, scoring="softmax", renormalize=True, weight_on="output", prefix="m.", expert_unit="silu",
                         router_bias=True)
    part.load({n: torch.as_tensor(v) for n, v in W.items()}, Runtime(torch.device(DEV), DT[dtype]))
    h = bf(rng.standard_normal((T, H)))
    want = pz.experts(h, W, "m.", {"experts": E, "top": top})
    for router_linear in (part.router_linear, None):        # logits by a product with the bias in it, or by the router kernel
        part.router_linear = router_linear
        got = part.forward(dev(h, DT[dtype]), None)
        if dtype == "float32":
            close(got, want, 3e-5, "mixture")
        else:       # a close call of the router moves a whole row: judge the typical row
            err = np.abs(got.float().cpu().numpy() - want).max(-1) / np.abs(want).max()
            assert float(np.median(err)) < 2e-2 and float((err > 6e-2).mean()) <= 0.05, f"median {np.median(err)}, worst {err.max()}"


def test_the_bias_alone_chooses():
    """Equal logits in front of the bias: it chooses the experts and weighs them."""
    from acvram_b200.kernels import ops
    T, E, top = 5, 6, 3
    z = torch.zeros((T, E), device=DEV)
    bias = torch.tensor([0.0, 3.0, -1.0, 3.0 - math.log(2.0), 0.5, -9.0], device=DEV)
    ids, w = torch.zeros(T * top, dtype=torch.int32, device=DEV), torch.zeros(T * top, device=DEV)
    ops.moe_route(torch.zeros((T, 8), device=DEV), torch.zeros((E, 8), device=DEV), None, top, True, True, ids, w, None, router_bias=bias)
    assert ids.view(T, top).cpu().tolist() == [[1, 3, 4]] * T
    got_ids, got_w = ids.clone(), w.clone()
    ops.moe_route(torch.zeros((T, 8), device=DEV), None, None, top, True, True, ids, w, None, logits=z + bias, experts=E)
    assert torch.equal(ids, got_ids) and torch.allclose(w, got_w)
    want = pz.choose(bias.cpu().double().numpy(), top)[1]
    close(w.view(T, top)[2], want, 1e-6, "weights")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,H,F", [(1, 64, 80), (33, 100, 37), (300, 128, 384)])
def test_dense_unit_with_gelu_in_the_product(T, H, F, dtype):
    from acvram_b200.parts.base import Runtime
    from acvram_b200.parts.feed_forward import DenseFF
    rng = np.random.default_rng(T + F)
    W = {"m.up": bf(1.5 * rng.standard_normal((F, H)) / math.sqrt(H)), "m.down": bf(rng.standard_normal((H, F)) / math.sqrt(F))}
    part = DenseFF(H, F, activation="gelu_tanh", prefix="m.")
    part.load({n: torch.as_tensor(v) for n, v in W.items()}, Runtime(torch.device(DEV), DT[dtype]))
    h = bf(rng.standard_normal((T, H)))
    close(part.forward(dev(h, DT[dtype]), None), pz.dense(h, W, "m."), 3e-5 if dtype == "float32" else 3e-2, "dense unit")
