"""Zogapel on the GPU: the engine against the plain implementation of tests/plain_zogapel.py.

Small configurations with random weights (tests/zogapel_util.py), logits asked at every position.  float32 runs must
agree with the float64 oracle to rounding, whatever the cut into steps, the batch, the pages or the state slots;
bfloat16 runs within what rounding does, judged by the typical position and by the far ones.
"""

from __future__ import annotations

import functools
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_zogapel as pz
import zogapel_util as zu
from conftest import ROOT
from test_lodalix_gpu import _read, ids_of, make_runner, mixed_schedule, play

pytestmark = pytest.mark.gpu

F32_BOUND = 3e-4        # float32 engine against the float64 oracle, per position (relative, see zu.row_errors)
# bfloat16: the median position, and the share of positions that may be further off than the bound (a router's close call
# sends a token to another expert)
BF16_MEDIAN, BF16_FAR, BF16_SHARE = 0.04, 0.15, 0.03


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("zogapel")
    return {w: zu.write_model(str(root / w), zu.config(w), seed=71 + i) for i, w in enumerate("ABCD")}


@functools.lru_cache(maxsize=None)
def oracle(folder: str, ids: tuple) -> np.ndarray:
    cfg, tensors = _read(folder)
    return pz.forward(cfg, tensors, list(ids))


def agree(folder, requests, got, dtype, what=""):
    errs = {r: zu.row_errors(got[r], oracle(folder, tuple(ids))) for r, ids in requests.items()}
    for r, err in errs.items():
        assert np.isfinite(err).all(), f"{what} {r}: not finite"
        if dtype == "float32":
            bad = np.nonzero(err > F32_BOUND)[0].tolist()
            assert not bad, f"{what} {r}: positions {bad[:8]} differ by {err[bad[:8]].tolist()}"
    if dtype == "bfloat16":
        # (a recurrence's output at a request's first token is v times one number, <q, k>, brought to unit RMS: where that is
        # nearly zero its rounding decides the sign, so first tokens are not judged)
        every = np.concatenate([e[1:] for e in errs.values() if len(e) > 1] or [np.zeros(1)])
        assert float(np.median(every)) < BF16_MEDIAN, f"{what}: median {float(np.median(every)):.4f}"
        assert float((every > BF16_FAR).mean()) <= BF16_SHARE, f"{what}: {int((every > BF16_FAR).sum())} of {every.size} far off, " \
            f"largest {float(every.max()):.3f}"


# --------------------------------------------------------------------------- whole prompts, layer by layer
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
def test_whole_prompts(folders, which, dtype):
    f = folders[which]
    runner = make_runner(f, dtype)
    requests = {f"w{n}": ids_of(f, n, n) for n in (1, 2, 3, 23, 150, 333)}     # the first tokens alone; page borders
    got = play(runner, requests, [{r: len(ids)} for r, ids in requests.items()])
    agree(f, requests, got, dtype, "whole")


@pytest.mark.parametrize("which", ["A", "C"])
def test_stream_after_every_layer(folders, which):
    f = folders[which]
    runner = make_runner(f, "float32")
    ids = ids_of(f, 61, 5)
    streams = []
    for blk in runner.model.blocks:
        def wrapped(x, delta, ctx, cache, orig=blk.forward):
            x, d = orig(x, delta, ctx, cache)
            y = d.tensor.double()               # the part's output joins behind its norm, in the next kernel
            y = y / (y.pow(2).mean(-1, keepdim=True) + d.eps).sqrt() * d.weight.double()
            streams.append((x.double() + y).cpu().numpy())
            return x, d
        blk.forward = wrapped
    play(runner, {"s": ids}, [{"s": len(ids)}])
    cfg, tensors = _read(f)
    want = []
    pz.forward(cfg, tensors, list(ids), streams=want)
    assert len(streams) == len(want) == len(cfg["layers"])
    for run, (g, w) in enumerate(zip(streams, want)):
        assert float(np.abs(g - w).max()) < 1e-4 * float(np.abs(w).max()), f"the stream leaves the oracle's after layer {run}"


# --------------------------------------------------------------------------- prefill against decoding, portions
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
def test_decoding_token_by_token(folders, which, dtype):
    """A prompt, then 120 tokens one by one, over page borders (16) and windows that pass over decoded tokens; in bfloat16
    through captured graphs.  A second request decodes from its second token on."""
    f = folders[which]
    runner = make_runner(f, dtype, graphs=dtype == "bfloat16")
    requests = {"d": ids_of(f, 37 + 120, 21), "e": ids_of(f, 1 + 30, 22)}
    steps = [{"d": 37}] + [{"d": 1}] * 120 + [{"e": 1}] * 31
    got = play(runner, requests, steps)
    agree(f, requests, got, dtype, "decode")
    if dtype == "bfloat16":
        assert runner.graph_launches > 0, "the decode steps did not replay a captured graph"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
def test_portions_of_any_size(folders, which, dtype):
    """Portions down to two tokens, longer than a block of the recurrence kernel (8 tokens) and no multiple of it, shorter than
    the convolution reaches, and single tokens between them (which take the step's kernel for portions or the one for
    single tokens)."""
    f = folders[which]
    runner = make_runner(f, dtype)
    ids = ids_of(f, 260, 31)
    sizes = [2, 3, 2, 17, 5, 31, 2, 70, 1, 7, 64, 2, 16, 1, 1, 1]
    sizes.append(len(ids) - sum(sizes))
    got = play(runner, {"p": ids}, [{"p": n} for n in sizes])
    agree(f, {"p": ids}, got, dtype, "portions")


def test_long_decoding_in_few_pages(folders):
    """A request of 500 tokens, 400 of them decoded one by one, in pages of 8: every layer of this model has a window (17, 40
    and 100 keys), so 16 pages are enough for it, and states and kept inputs run on for hundreds of steps."""
    f = folders["A"]
    runner = make_runner(f, "float32", pages=18, page_size=8, max_requests=2)
    ids = ids_of(f, 500, 77)
    got = play(runner, {"long": ids}, [{"long": 30}, {"long": 11}, {"long": 2}, {"long": 30}, {"long": 27}] + [{"long": 1}] * 400)
    agree(f, {"long": ids}, got, "float32", "long")


# --------------------------------------------------------------------------- batches, pages and slots used again
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
def test_mixed_batches_in_a_small_pool(folders, which, dtype):
    """Seven unequal requests, three live at a time, portions beside single tokens, with rows of the block tables, pages
    and state slots for three requests: all are used again (the state of a slot's former request must be gone), and
    every request must come out as it does alone."""
    f = folders[which]
    lengths = (90, 14, 131, 1, 57, 160, 33)
    requests = {f"m{i}": ids_of(f, n, 40 + i) for i, n in enumerate(lengths)}
    pages = 3 * (-(-160 // 16))
    runner = make_runner(f, dtype, pages=pages, max_requests=3, graphs=dtype == "bfloat16")
    got = play(runner, requests, mixed_schedule(requests, 7, 3))
    agree(f, requests, got, dtype, "mixed")
    assert all(g.pool.num_free == pages for g in runner.manager.paged_groups)
    assert all(g.num_free == 3 for g in runner.manager.state_groups)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim,rot", [(24, 8), (64, 16)])
def test_a_far_key_decides(tmp_path, dtype, dim, rot):
    """One attention layer alone without a window and with a sharp softmax: position 600 must find the keys of the first
    tokens.  The oracle's logits without those tokens differ from the true ones by more than the bounds, so a kernel that
    lost them fails."""
    cfg = zu.model(128, 64, [zu.layer(zu.attention(2, 1, dim, rot, 0, 1e4, (4.0, 128, 8.0, 1.0), scale=4.0 * dim ** -0.5), None)], 1e-5)
    f = zu.write_model(str(tmp_path / "far"), cfg, 5)
    ids = ids_of(f, 640, 99)
    runner = make_runner(f, dtype, pages=48)
    got = play(runner, {"far": ids}, [{"far": 590}] + [{"far": 1}] * 50)
    agree(f, {"far": ids}, got, dtype, "far")
    cut = oracle(f, tuple(ids[48:]))                       # the same tokens without the first three pages
    err = zu.row_errors(cut[-40:], oracle(f, ids)[-40:])
    assert float((err > BF16_FAR).mean()) > 0.03, "the far keys do not matter in this test: it shows nothing"


def _shouting(cfg, seed):
    """Weights in which token 63 shouts: its embedding is the stream's element 0 alone, which no other token has."""
    w = zu.random_weights(cfg, seed)
    w["embed"][:, 0] = 0.0
    w["embed"][63] = 0.0
    w["embed"][63, 0] = 1.0
    for i in range(len(cfg["layers"])):
        w[f"l{i}.norm1"][0] = 0.0
    return w


def _places(f, places, n, steps_list, dtype="float32"):
    """A shouting token at each of ``places`` ({place: whether the last position sees it}), in several cuts into steps."""
    c, tensors = zu.read_folder(f)
    base = [t % 60 for t in ids_of(f, n, 4)]
    quiet = pz.forward(c, tensors, base)[-1]
    for place, seen in places.items():
        ids = list(base)
        ids[place] = 63
        want = pz.forward(c, tensors, ids)
        moved = float(zu.row_errors(want[-1:], quiet[None])[0])
        assert moved > 0.05 if seen else moved < 1e-9, f"the oracle itself: place {place} moves the last logits by {moved}"
        for steps in steps_list:
            runner = make_runner(f, dtype, pages=16)
            got = play(runner, {"r": ids}, steps)["r"]
            err = zu.row_errors(got, want)
            if dtype == "float32":
                assert float(err.max()) < F32_BOUND, f"place {place}, steps {steps[:2]}"
            else:
                assert float(err[-1]) < (0.5 * moved if seen else 0.025), f"place {place}, steps {steps[:2]}: {float(err[-1])}"


@pytest.mark.parametrize("dtype,dim", [("float32", 16), ("float32", 64), ("bfloat16", 64), ("bfloat16", 128), ("bfloat16", 48)])
@pytest.mark.parametrize("window", [1, 5, 16, 17, 31])
def test_a_key_at_the_windows_edge(tmp_path, window, dtype, dim):
    """One attention layer alone.  The shouting token's key, its own value, stands out.  It is placed as the last key inside
    the window, the first one outside it, first, last, and on both sides of page borders (pages of 16), for a prompt, for
    decoded tokens and for portions."""
    cfg = zu.model(64, 32, [zu.layer(zu.attention(2, 1, dim, 8, window, 1e3, (2.0, 64, 8.0, 1.0), scale=0.02), None)], 1e-5)
    w = _shouting(cfg, 3)
    w["l0.mix.k"][:, 0] = 6.0
    w["l0.mix.g"][:] = 0.0
    w["l0.mix.o"] = w["l0.mix.o"].abs() * 0.25 + w["l0.mix.o"]
    f = zu.write_model(str(tmp_path / "edge"), cfg, 0, w)
    n = 39
    places = {p: n - 1 - p < window for p in {0, n - 1 - window, n - window, n - 1, 15, 16, 31, 32} if p >= 0}
    _places(f, places, n, ([{"r": n}], [{"r": n - 1}, {"r": 1}], [{"r": n - 3}, {"r": 1}, {"r": 2}],
                           [{"r": 15}, {"r": 2}, {"r": n - 20}, {"r": 2}, {"r": 1}]), dtype)


def test_a_state_remembers_the_first_token(tmp_path):
    """One recurrence alone that does not decay: what the first token wrote weighs at the end, 200 tokens on, whatever the cut;
    and one that keeps nothing has only the last tokens left."""
    K = 3
    cfg = zu.model(64, 32, [zu.layer(zu.delta(2, 1, 32, 8, K), None)], 1e-5)
    w = _shouting(cfg, 9)
    w["l0.mix.A_log"][:] = -30.0
    w["l0.mix.b"][:] = -0.2 * w["l0.mix.b"].abs()           # small steps
    w["l0.mix.b"][:, 0] = 4.0                               # but the shouting token writes in full
    w["l0.mix.v"][:, 0] = 30.0
    f = zu.write_model(str(tmp_path / "keeps"), cfg, 0, w)
    n = 200
    cuts = ([{"r": n}], [{"r": 33}, {"r": 2}, {"r": n - 36}, {"r": 1}], [{"r": 100}] + [{"r": 1}] * 100)
    c, tensors = zu.read_folder(f)
    base = [t % 60 for t in ids_of(f, n, 4)]
    first = list(base)
    first[0] = 63
    moved = float(zu.row_errors(pz.forward(c, tensors, first)[-1:], pz.forward(c, tensors, base)[-1:])[0])
    assert moved > 10 * F32_BOUND, f"the oracle itself: the first token moves the last logits by {moved}"
    for steps in cuts:
        got = play(make_runner(f, "float32", pages=16), {"r": first}, steps)["r"]
        assert float(zu.row_errors(got, pz.forward(c, tensors, first)).max()) < F32_BOUND
    w["l0.mix.A_log"][:] = 6.0                              # keeps nothing: the convolution's reach is all that is left
    w["l0.mix.dt_bias"][:] = 4.0
    f = zu.write_model(str(tmp_path / "forgets"), cfg, 0, w)
    _places(f, {0: False, n - K - 1: False, n - K: True, n - 1: True}, n, cuts)


# --------------------------------------------------------------------------- the entry points
@pytest.mark.parametrize("which", ["A", "D"])
def test_greedy_generation_through_the_engine(folders, which):
    from acvram_b200 import Engine, SamplingParams
    f = folders[which]
    cfg, tensors = _read(f)
    prompts = [list(ids_of(f, 19, 1)), list(ids_of(f, 70, 2)), list(ids_of(f, 3, 3))]
    want = [pz.greedy(cfg, tensors, p, 12) for p in prompts]
    for dtype in ("float32", "bfloat16"):
        engine = Engine(f, dtype, max_batch_size=3, max_model_len=128, page_size=16, num_pages=24, token_budget=48,
                        device="cuda:0")
        got = engine.generate_batch(prompts, SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True))
        assert not engine.stats.failed_steps, engine.last_error
        if dtype == "float32":
            assert got == want
        else:
            for p, g in zip(prompts, got):      # the first token is one of the oracle's best (a close call may go either way)
                row = oracle(f, tuple(p))[-1]
                assert len(g) == 12 and row[g[0]] > row.max() - 0.3 * row.std()


def test_trace_run_program(folders, tmp_path):
    f = folders["C"]
    ids = ids_of(f, 45, 8)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": list(ids[:30]), "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": list(ids[30:44]), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": [ids[44]], "want": [0]},
                                     {"id": "y", "tokens": list(ids[:7]), "want": [6]}], "end": ["x", "y"]}]
    out = tmp_path / "out"
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", f, "--dtype", "float32", "--out", str(out),
                           "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n", text=True,
                          capture_output=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not (out / "1.f32").exists()
    full = oracle(f, tuple(ids))
    vocab = full.shape[1]
    a = np.fromfile(out / "0.f32", dtype="<f4").reshape(-1, vocab)
    b = np.fromfile(out / "2.f32", dtype="<f4").reshape(-1, vocab)
    assert float(zu.row_errors(a, full[[0, 29]]).max()) < F32_BOUND
    assert float(zu.row_errors(b, np.stack([full[44], full[6]])).max()) < F32_BOUND


@pytest.mark.parametrize("ahead", [False, True])
def test_preemption_starts_the_states_anew(folders, ahead):
    """One layer keeps every key, so a pool of 7 pages cannot hold three requests of 55 tokens: requests are preempted and
    computed again from their first token, in state slots that others have used meanwhile.  States and kept inputs must
    start at zero again: the greedy tokens stay the oracle's."""
    from acvram_b200 import Engine, SamplingParams
    f = folders["C"]
    cfg, tensors = _read(f)
    prompts = [list(ids_of(f, n, 500 + n)) for n in (20, 25, 18)]
    want = [pz.greedy(cfg, tensors, p, 30) for p in prompts]
    engine = Engine(f, "float32", max_batch_size=3, max_model_len=128, page_size=16, num_pages=7, token_budget=16,
                    device="cuda:0", run_ahead=ahead)
    got = engine.generate_batch(prompts, SamplingParams(temperature=0.0, max_tokens=30, ignore_eos=True))
    assert not engine.stats.failed_steps, engine.last_error
    assert engine.stats.preempted > 0, "the pool was meant to be too small"
    assert got == want
    engine.runner.manager.check()
    assert all(g.num_free == g.max_requests for g in engine.runner.manager.state_groups)
