"""The kernels of the Lodalix parts one by one, each against the oracle's function of the same mechanism on the same
(bfloat16-rounded) inputs: a request's tokens cut into steps of several sizes (down to one and two tokens) against the
whole sequence, states carried in slots that are not the requests' indices, kept rows in pages handed out in any order,
sinks beside and far above the scores, branches on both sides of their clamps."""

from __future__ import annotations

import math

import numpy as np
import pytest
import torch

import plain_lodalix as pl
from test_nizedra_kernels_gpu import paged_case
from test_vadelix_kernels_gpu import DEV, DT, batches, bf, close, dev, i32, step_arrays

pytestmark = pytest.mark.gpu

CUTS = ([1] * 9, [2, 2, 2, 2, 1], [9], [3, 1, 5], [1, 8], [7, 2], [4, 5])


# --------------------------------------------------------------------------- the generalized delta rule
def delta_weights(rng, width, H, D, L, decay_at=-1.0):
    W = {"x." + n: bf(1.2 * rng.standard_normal((H * D, width)) / math.sqrt(width)) for n in "rkvga"}
    W.update({"x.a.b": bf(rng.standard_normal(H * D)), "x.w1": bf(1.5 * rng.standard_normal((L, width)) / math.sqrt(width)),
              "x.w2": bf(1.5 * rng.standard_normal((H * D, L)) / math.sqrt(L)), "x.w0": bf(decay_at + rng.standard_normal(H * D)),
              "x.norm": bf(1.0 + 0.2 * rng.standard_normal(H * D)), "x.o": np.eye(H * D)})
    return W


def delta_proj(h, W, pad):
    """The input product of the tokens h, as the part stacks it (with ``pad`` columns behind)."""
    cols = [h @ W["x." + n].T for n in "rkv"] + [h @ W["x.a"].T + W["x.a.b"], h @ W["x.g"].T, h @ W["x.w1"].T,
                                                 np.zeros((h.shape[0], pad))]
    return dev(np.concatenate(cols, axis=1))


def blocks(q_lens):
    from acvram_b200.kernels import ops
    arrays, values = ops.delta_work(q_lens)
    return {**{k: i32(v) for k, v in arrays.items()}, **values}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,D,L", [(2, 8, 3), (1, 4, 1), (3, 10, 5), (2, 16, 8), (3, 20, 7), (2, 32, 16), (5, 48, 4), (2, 64, 32),
                                   (1, 100, 9), (2, 128, 12), (1, 200, 6), (1, 300, 5)])
def test_delta_over_steps(H, D, L, dtype):
    """Three requests side by side, cut differently, their states in slots 4, 0 and 2: portions through prepare, recurrence
    and gate, steps of single tokens through the one-launch kernel where the head allows it."""
    from acvram_b200.kernels import ops
    rng = np.random.default_rng(H * 1000 + D)
    width, I, pad = 40, H * D, 3
    lengths, slots_of = (9, 9, 9), (4, 0, 2)
    W = delta_weights(rng, width, H, D, L)
    hs = [bf(rng.standard_normal((n, width))) for n in lengths]
    state = torch.zeros((5, H, D, D), device=DEV)
    got = [np.zeros((n, I)) for n in lengths]
    w2t, w0, nw = dev(W["x.w2"].T.copy()), dev(W["x.w0"]), dev(W["x.norm"])
    for cuts in ((CUTS[0], CUTS[0], CUTS[0]), (CUTS[1], CUTS[2], CUTS[5]), (CUTS[3], CUTS[4], CUTS[6])):
        state.zero_()
        for step in batches(lengths, cuts):
            cu, _ = step_arrays(step)
            proj = delta_proj(np.concatenate([hs[r][a:a + c] for r, a, c in step]), W, pad)
            T = proj.shape[0]
            wide = torch.full((T, I + 5), 7.0, device=DEV, dtype=DT[dtype])       # the heads land in columns of wider rows
            ops.general_delta(proj, w2t, w0, nw, 1e-5, state, i32([slots_of[r] for r, _, _ in step]), cu, len(step),
                              max(c for _, _, c in step), wide[:, :I], H, D, L, blocks([c for _, _, c in step]))
            assert bool((wide[:, I:] == 7.0).all())
            at = 0
            for r, a0, c in step:
                got[r][a0:a0 + c] = wide[at:at + c, :I].float().cpu().numpy()
                at += c
        for r in range(3):
            want = pl.general_delta(hs[r], W, "x.", {"heads": H, "dim": D}, 1e-5)
            close(got[r], want, 1e-4 if dtype == "float32" else 1e-2, f"request {r}, cuts {cuts[r]}")
        assert float(state[1].abs().max()) == 0.0 == float(state[3].abs().max())      # slots of nobody


@pytest.mark.parametrize("D", [12, 64])
def test_a_long_portion_equals_token_by_token(D):
    """300 tokens of one request as one portion (many blocks of the kernel), one by one (the one-launch kernel) and cut
    around a single token (blocks of eight tokens begin anywhere); decays close to 1 and few removals, so that the first tokens still weigh at the end."""
    from acvram_b200.kernels import ops
    rng = np.random.default_rng(D)
    n, H, L, width = 300, 2, 4, 32
    W = delta_weights(rng, width, H, D, L, decay_at=-6.0)
    W["x.a.b"] = W["x.a.b"] - 4.0
    h = bf(rng.standard_normal((n, width)))
    w2t, w0, nw = dev(W["x.w2"].T.copy()), dev(W["x.w0"]), dev(W["x.norm"])
    want = pl.general_delta(h, W, "x.", {"heads": H, "dim": D}, 1e-5)
    short = pl.general_delta(h[40:], W, "x.", {"heads": H, "dim": D}, 1e-5)
    assert float(np.abs(short[-1] - want[-1]).max()) > 1e-2 * float(np.abs(want[-1]).max()), "the first tokens do not matter here"
    for cuts in ([n], [1] * n, [130, 1, 169], [31, 33, 32, 8, 196]):
        state = torch.zeros((2, H, D, D), device=DEV)
        got = torch.empty((n, H * D), device=DEV)
        at = 0
        for c in cuts:
            proj = delta_proj(h[at:at + c], W, 0)
            ops.general_delta(proj, w2t, w0, nw, 1e-5, state, i32([1]), i32([0, c]), 1, c, got[at:at + c], H, D, L, blocks([c]))
            at += c
        close(got, want, 2e-4, f"cuts {cuts[:3]}")


# --------------------------------------------------------------------------- kept rows, queries
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("halves", [False, True])
@pytest.mark.parametrize("H,D,R,KR", [(3, 8, 6, 20), (1, 16, 2, 33), (8, 64, 64, 128)])
def test_kept_rows_and_queries(H, D, R, KR, halves, dtype):
    """A token's kept row in its page and the heads' rotated query parts, for both pairings with scaled frequencies; and
    queries alone, for a layer that reads another one's rows (the pages stay as they are)."""
    from acvram_b200.kernels import ops
    from acvram_b200.parts.base import Runtime
    from acvram_b200.parts.position import Rotary
    rng = np.random.default_rng(H + R)
    T, page, t = 21, 8, DT[dtype]
    rot = {"base": 700.0, "dims": R, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}}
    pos_part = Rotary(1, R, 700.0, 64, scaling=(4.0, 64, 8.0, 1.0) if halves else None, exact=True)
    pos_part.load({}, Runtime(torch.device(DEV), t))
    q, kv, w = bf(rng.standard_normal((T, H, D + R))), bf(rng.standard_normal((T, KR + R))), bf(1.0 + 0.2 * rng.standard_normal(KR))
    table = torch.tensor([[-1, -1, -1], [4, 1, 2]], dtype=torch.int32, device=DEV)
    for own in (True, False):
        pages = torch.full((6, 1, page, KR + R), 9.0, device=DEV, dtype=t)
        met = torch.full((T, H * (KR + R)), 7.0, device=DEV, dtype=t)
        ops.latent_prepare(dev(q.reshape(T, -1), t), met, dev(kv, t) if own else None, dev(w) if own else None, 1e-5,
                           pos_part.rotary_table(), i32(range(T)), i32([0] * T), table if own else None, pages if own else None,
                           H, D, R, KR, table_rows=i32([1]), rotate_half=halves)
        m = met.view(T, H, KR + R)
        close(m[:, :, KR:], pl.rotate(q[:, :, D:], rot, halves), 1e-5 if dtype == "float32" else 1e-2, "queries")
        assert bool((m[:, :, :KR] == 7.0).all())
        if own:
            rows = pages[torch.tensor([4, 1, 2])].reshape(3 * page, KR + R)[:T]
            want = np.concatenate([pl.unit_rms(kv[:, :KR], 1e-5) * w, pl.rotate(kv[:, KR:], rot, halves)], axis=1)
            close(rows, want, 1e-5 if dtype == "float32" else 1e-2, "kept rows")
        else:
            assert bool((pages == 9.0).all())


SINK_CASES = [
    # NH  ROW  KR  page  lens              q_lens
    (8, 144, 128, 64, [200, 150, 97], [130, 1, 2]),             # a portion, a decoded token, two tokens in one launch
    (3, 72, 48, 16, [90, 21], [17, 1]),
    (16, 576, 512, 64, [400, 300, 64], [150, 1, 1]),            # four warps share a row group
    (80, 320, 256, 16, [60, 40], [9, 1]),                       # head blocks
    (16, 144, 128, 16, [900, 40, 1300], [1, 1, 1]),             # one-token requests whose rows several CTAs share
    (20, 576, 512, 64, [700, 64, 65, 3], [1, 1, 1, 1]),         # more heads than a CTA's 16, a tile's edge, a few keys
    (5, 72, 48, 8, [130, 9], [1, 1]),                           # small pages; rows that end inside a 64-element piece
    (6, 200, 136, 128, [300, 129], [1, 1]),                     # pages of two tiles
]


@pytest.mark.parametrize("case", SINK_CASES, ids=lambda c: f"h{c[0]}row{c[1]}kr{c[2]}")
def test_sinks_over_kept_rows(case):
    """Sinks far below, beside and far above the scores, in the generic and the tensor-core kernel, whole rows and
    rows shared among CTAs, with one key planted so that its score stands out."""
    from acvram_b200.kernels import ops
    NH, ROW, KR, page, lens, q_lens = case
    ctx, work, table, k, _, T = paged_case(1, ROW, 8, page, lens, q_lens, 31 + NH, torch.bfloat16)
    g = torch.Generator().manual_seed(NH + ROW)
    q = torch.randn(T, NH * ROW, generator=g)
    q = (q / q.pow(2).mean(-1, keepdim=True).sqrt()).to(torch.bfloat16).to(DEV)
    # request 0's key at a page's last place is the first head's query of its last token: one score of ROW * scale
    place = min(page - 1, lens[0] - 2)
    k[table[0, place // page].item(), 0, place % page] = q[q_lens[0] - 1, :ROW]
    scale = ROW ** -0.5 * 3.0
    sinks = torch.tensor([(-30.0, 0.0, 2.0, 40.0)[h % 4] for h in range(NH)])
    want = np.zeros((T, NH, KR))
    t0 = 0
    for b, (n, ql) in enumerate(zip(lens, q_lens)):
        js = torch.arange(n)
        rows = k.cpu().double()[table[b].long().cpu()[js // page], 0, js % page].numpy()
        qq = q[t0:t0 + ql].cpu().double().view(ql, NH, ROW).numpy()
        for h in range(NH):
            s = np.full((n, n), -np.inf)
            s[n - ql:] = qq[:, h] @ rows.T * scale
            s[:n - ql] = 0.0
            want[t0:t0 + ql, h] = pl.causal_weights(s, float(sinks[h]))[n - ql:] @ rows[:, :KR]
        t0 += ql
    plain = max(abs(want).max(), 1e-9)
    sd = sinks.to(DEV)
    out = torch.zeros((T, NH * KR), device=DEV)
    ops.attention_latent(q.float(), out, k.float(), ctx, table, NH, ROW, KR, scale, sinks=sd)
    assert float(np.abs(out.cpu().double().numpy().reshape(T, NH, KR) - want).max()) < 2e-4 * plain
    assert ops.attention_latent_tc_takes(torch.bfloat16, NH, ROW, KR)
    out = torch.full((T, NH * KR), 7.0, device=DEV, dtype=torch.bfloat16)
    ops.attention_latent(q, out, k, ctx, table, NH, ROW, KR, scale, work=work, sinks=sd)
    assert float(np.abs(out.cpu().double().numpy().reshape(T, NH, KR) - want).max()) < 2e-2 * plain


@pytest.mark.parametrize("window", [0, 70])
def test_one_token_requests_over_kept_rows_under_a_window(window):
    """The kernel for one-token requests beside a padded slot of a captured batch (no context): zeros come out, and the
    others are as the dense sums say, with and without a window."""
    from acvram_b200.kernels import ops
    NH, ROW, KR, page, lens = 7, 144, 128, 16, [200, 71, 70, 1]
    ctx, work, table, k, _, T = paged_case(1, ROW, 8, page, lens, [1, 1, 1, 1], 8, torch.bfloat16)
    q = torch.randn(T, NH * ROW, generator=torch.Generator().manual_seed(4)).to(torch.bfloat16).to(DEV)
    ctx.kv_len[3] = 0
    out = torch.full((T, NH * KR), 7.0, device=DEV, dtype=torch.bfloat16)
    ops.attention_latent(q, out, k, ctx, table, NH, ROW, KR, 0.1, window, work=work)
    assert float(out[3].abs().max()) == 0.0
    for b, n in enumerate(lens[:3]):
        js = torch.arange(max(0, n - window) if window else 0, n)
        rows = k.cpu().double()[table[b].long().cpu()[js // page], 0, js % page].numpy()
        s = q[b].cpu().double().view(NH, ROW).numpy() @ rows.T * 0.1
        w = np.exp(s - s.max(-1, keepdims=True))
        close(out[b].view(NH, KR), (w / w.sum(-1, keepdims=True)) @ rows[:, :KR], 2e-2, f"request {b}")


@pytest.mark.parametrize("H,D,R,DV,KR,page,gated", [(3, 16, 8, 24, 48, 16, True), (4, 64, 64, 128, 128, 64, False), (2, 7, 2, 9, 33, 8, True),
                                                    (5, 32, 32, 64, 64, 16, False)])
def test_written_out_keys_and_values(H, D, R, DV, KR, page, gated):
    """A step of two portions and a one-token request, the portions' contexts longer than their tokens: keys and values
    written out from the pages (pages in any order), attention over them, the heads gated into columns of wider rows, the
    one-token request picked out of the queries.  One key at a page's end is planted so that its score stands out."""
    from acvram_b200.kernels import ops
    rng = np.random.default_rng(H * 10 + D)
    HD, ROW = (64 if max(D + R, DV) <= 64 else 128), KR + R
    lens, q_lens = [190, 33, 260], [150, 1, 77]
    ctx, work, table, pages, _, T = paged_case(1, ROW, 8, page, lens, q_lens, 3 + H, torch.bfloat16)
    arrays, values = ops.latent_context_work(q_lens, lens)
    assert values["n_pages"] == 2 + 3 and arrays["table"].reshape(3, -1).tolist() == [[0, 1, -1], [-1, -1, -1], [2, 3, 4]]
    ex = {**{k: i32(v) for k, v in arrays.items()}, **values}
    uk, uv = bf(rng.standard_normal((H, D, KR)) / math.sqrt(KR)), bf(rng.standard_normal((H, DV, KR)) / math.sqrt(KR))
    q = bf(rng.standard_normal((T, H, D + R)))
    rows = [pages.cpu().double()[table[b].long().cpu()[torch.arange(n) // page], 0, torch.arange(n) % page].numpy() for b, n in enumerate(lens)]
    place = lens[2] // page * page - 1
    rows[2][place, KR:] = q[-1, 0, D:] * 3.0 / math.sqrt(R)
    pages[table[2, place // page].item(), 0, place % page] = dev(rows[2][place], torch.bfloat16)
    rows[2][place] = pages[table[2, place // page].item(), 0, place % page].cpu().double().numpy()
    scale = 1.5 * (D + R) ** -0.5
    z, sinks = bf(rng.standard_normal((T, H * DV))), bf(rng.standard_normal(H))
    want = np.zeros((T, H, DV))
    t0 = 0
    for b, (n, ql) in enumerate(zip(lens, q_lens)):
        for h in range(H):
            keys = np.concatenate([rows[b][:, :KR] @ uk[h].T, rows[b][:, KR:]], axis=1)
            s = np.zeros((n, n))
            s[n - ql:] = q[t0:t0 + ql, h] @ keys.T * scale
            want[t0:t0 + ql, h] = pl.causal_weights(s, float(sinks[h]))[n - ql:] @ (rows[b][:, :KR] @ uv[h].T)
        t0 += ql
    want = want.reshape(T, -1) * (pl.sigmoid(z) if gated else 1.0)
    qx = torch.zeros((T, H, HD), device=DEV, dtype=torch.bfloat16)
    qx[:, :, :D + R] = dev(q, torch.bfloat16)
    qx = qx.view(T, -1)
    got_rows = ops.latent_context(pages, ctx, table, ex, ROW)
    assert torch.equal(got_rows[:lens[0]].double().cpu(), torch.as_tensor(rows[0])) and float(got_rows[lens[0]:256].abs().max()) == 0.0
    w = torch.cat([dev(uk.reshape(-1, KR), torch.bfloat16), dev(uv.reshape(-1, KR), torch.bfloat16)])
    kv = got_rows[:, :KR] @ w.t()
    kp, vp = ops.latent_pack(kv, got_rows, H, D, R, DV, KR, HD)
    o = torch.full((T, H * HD), 7.0, device=DEV, dtype=torch.bfloat16)
    sd = dev(sinks)
    ops.attention_tc(qx, o, kp, vp, work["tile_seq"], work["tile_q0"], work["n_tiles"], ctx.cu_q, ctx.kv_len,
                     ex["table"].view(-1, ex["width"]), H, H, HD, scale, 0, sinks=sd)
    out = torch.full((T, H * DV + 5), 7.0, device=DEV, dtype=torch.bfloat16)
    gate = dev(z, torch.bfloat16) if gated else None
    ops.heads_gated(o, HD, gate, None, out[:, :H * DV], H, DV)
    met = torch.zeros((1, H * ROW), device=DEV, dtype=torch.bfloat16)
    plain = ops.latent_pick(qx, HD, work["dec_tokens"], 1, met, H, D, R, KR)
    assert torch.equal(plain[0].double().cpu(), torch.as_tensor(q[150, :, :D])) and torch.equal(met.view(H, ROW)[:, KR:].double().cpu(), torch.as_tensor(q[150, :, D:]))
    one = dev(want[150:151].reshape(1, -1) if not gated else (want[150:151] / pl.sigmoid(z[150:151])).reshape(1, -1), torch.bfloat16)
    ops.heads_gated(one, DV, gate, work["dec_tokens"], out[:, :H * DV], H, DV)
    close(out[:, :H * DV], want, 2.5e-2, "heads")
    assert bool((out[:, H * DV:] == 7.0).all())


# --------------------------------------------------------------------------- gated per-head products, the clamped unit, the block
@pytest.mark.parametrize("T,B,K,N,pad", [(70, 3, 64, 96, 8), (1, 16, 64, 128, 0), (33, 2, 12, 20, 3), (130, 5, 22, 9, 0)])
def test_per_head_products_with_a_gate(T, B, K, N, pad):
    from acvram_b200.kernels import ops
    rng = np.random.default_rng(T + K)
    a, w, z = bf(rng.standard_normal((T, B, K))), bf(rng.standard_normal((B, N, K)) / math.sqrt(K)), bf(2.0 * rng.standard_normal((T, B * N + pad)))
    want = np.einsum("tbk,bnk->tbn", a, w) * pl.sigmoid(z[:, pad:].reshape(T, B, N))
    for dtype, tol in (("bfloat16", 1e-2), ("float32", 1e-5)):
        out = torch.full((T, B * N + pad), 7.0, device=DEV, dtype=DT[dtype])
        gate = dev(z, DT[dtype])[:, pad:].unflatten(1, (B, N))
        ops.gemm_batched(dev(a, DT[dtype]), dev(w, DT[dtype]), out[:, :B * N].unflatten(1, (B, N)), gate=gate)
        close(out[:, :B * N].unflatten(1, (B, N)), want, tol, dtype)
        assert bool((out[:, B * N:] == 7.0).all())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,H,F", [(1, 64, 80), (5, 100, 60), (33, 96, 200), (130, 128, 72), (300, 128, 384), (600, 512, 1024)])
def test_clamped_unit_with_biases(T, H, F, dtype):
    """The gated unit with its clamps and biases: in the products' epilogue with tokens on the tensor core's columns (few)
    and rows (many), and outside it (rows that are no 16-byte pieces, float32); both branches pass their limits."""
    from acvram_b200.parts.base import Runtime
    from acvram_b200.parts.feed_forward import SwiGLU
    rng = np.random.default_rng(T + F)
    names = {r + b: r + s for r in ("gate", "up", "down") for b, s in (("", ""), (".bias", ".b"))}
    W = {"m.gate": bf(1.5 * rng.standard_normal((F, H)) / math.sqrt(H)), "m.up": bf(1.5 * rng.standard_normal((F, H)) / math.sqrt(H)),
         "m.down": bf(rng.standard_normal((H, F)) / math.sqrt(F)), "m.gate.b": bf(rng.standard_normal(F)),
         "m.up.b": bf(rng.standard_normal(F)), "m.down.b": bf(rng.standard_normal(H))}
    part = SwiGLU(H, F, prefix="m.", bias=True, names=names, activation="swish_clamped", limit=1.25, alpha=1.702)
    part.load({n: torch.as_tensor(v) for n, v in W.items()}, Runtime(torch.device(DEV), DT[dtype]))
    h = bf(rng.standard_normal((T, H)))
    pre = h @ W["m.gate"].T + W["m.gate.b"]
    assert float((pre > 1.25).mean()) > 0.05 and float((pre < -1.25).mean()) > 0.05
    close(part.forward(dev(h, DT[dtype]), None), pl.clamped_unit(h, W, "m.", 1.25), 3e-5 if dtype == "float32" else 2e-2, "clamped unit")
    wide = torch.full((T, F + 24), 7.0, device=DEV, dtype=DT[dtype])         # the inner columns land in wider rows
    part.inner(dev(h, DT[dtype]), None, wide[:, 16:16 + F])
    u = np.clip(h @ W["m.up"].T + W["m.up.b"], -1.25, 1.25)
    g = np.minimum(pre, 1.25)
    close(wide[:, 16:16 + F], g * pl.sigmoid(1.702 * g) * (u + 1.0), 3e-5 if dtype == "float32" else 2e-2, "inner columns")
    assert bool((wide[:, :16] == 7.0).all()) and bool((wide[:, 16 + F:] == 7.0).all())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_parallel_block_of_other_parts(dtype):
    """The block arrangement with parts of other designs: grouped-query attention beside a plain gated unit.  Its output is
    the sum of the two parts' own outputs on the same normed input."""
    from acvram_b200.cache import CacheManager, CacheStorage
    from acvram_b200.cache.manager import CachePlan
    from acvram_b200.engine.batch import BatchBuilder, StepEntry
    from acvram_b200.parts.base import CacheView, Runtime
    from acvram_b200.parts.blocks import ParallelBlock
    from acvram_b200.parts.plan import LayerSpec, PartSpec
    W, t = 64, DT[dtype]
    attn = PartSpec("attention", {"num_heads": 4, "num_kv_heads": 2, "head_dim": 16, "bias": False,
                                  "position": PartSpec("rotary", {"dim": 16, "theta": 1e4, "max_positions": 128})})
    blk = ParallelBlock(LayerSpec("", "parallel", attn, PartSpec("swiglu", {"intermediate_size": 88, "bias": False}),
                                  PartSpec("rmsnorm", {"eps": 1e-6}), norm_prefixes=("n.", "n.")), W)
    g = torch.Generator().manual_seed(2)
    tensors = {n: (torch.randn(need.shape, generator=g) * (W ** -0.5 if len(need.shape) > 1 else 0.1)).to(torch.bfloat16)
               for n, need in blk.tensor_needs().items()}
    blk.load(tensors, Runtime(torch.device(DEV), t))
    manager = CacheManager(CachePlan([blk.cache_need()]), 16, 8, 2)
    storage = CacheStorage(manager, DEV, t, 64)
    builder = BatchBuilder(manager, storage, DEV, 100, 64, {"attention": blk.mixer})
    manager.admit("r")
    manager.grow("r", 30)
    ctx = builder.build([StepEntry("r", list(range(30)), (29,))], [0])
    view = CacheView(0, True, *storage.pages(0))
    x = torch.randn(30, W, generator=g).to(DEV)
    _, delta = blk.forward(x.clone(), None, ctx, view)
    h = blk.input_norm.forward(x.clone(), None, out_dtype=t)
    want = blk.mixer.forward(h, ctx, view).double() + blk.feed_forward.forward(h, ctx).double()
    assert delta.dtype == torch.float32
    close(delta, want.cpu().numpy(), 1e-5 if dtype == "float32" else 1.5e-2, "the joint product")
