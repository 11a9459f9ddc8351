#!/usr/bin/env python3
"""Headline measurement: decode tokens/s of a Qwen3-8B-shaped model on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference]

The model has the layer sizes of Qwen3-8B (36 layers, hidden 4096, 32 query and
8 key/value heads of 128, intermediate 12288, vocabulary 151936, rope theta 1e6,
eps 1e-6, untied head) with random weights N(0, 0.02) in bfloat16; the default
run decodes a batch of 8 requests that each hold a 2048-token synthetic context
in a paged bfloat16 cache (pages of 16 tokens, as the baseline's configuration has them).  A step is one decode step of the whole
batch.  One JSON line is printed: ``value`` is decoded tokens per second timed on
the device over exactly K steps after W warm-up steps; ``e2e`` is the same through
``Engine.step()`` with host token ids in and out; ``prefill`` is one 2048-token
prompt; ``roofline`` is the decode step's necessary bytes over its time; ``points``
holds batch 1 and 64.  This program measures one GPU: for --gpus N > 1 it says so
and exits with 2.
"""

from __future__ import annotations

import argparse
import json
import os
import sys
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

QWEN3_8B = dict(vocab_size=151936, hidden_size=4096, intermediate_size=12288, num_hidden_layers=36,
                num_attention_heads=32, num_key_value_heads=8, head_dim=128, rms_norm_eps=1e-6, rope_theta=1000000.0,
                max_position_embeddings=40960, tie_word_embeddings=False)
# the larger shapes that the baseline's configurations name, for `--shape`; the default run is the 8B shape
SHAPES = {
    "8b": QWEN3_8B,
    "14b": {**QWEN3_8B, "hidden_size": 5120, "intermediate_size": 17408, "num_hidden_layers": 40, "num_attention_heads": 40},
    "32b": {**QWEN3_8B, "hidden_size": 5120, "intermediate_size": 25600, "num_hidden_layers": 64, "num_attention_heads": 64},
}
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0}


def peaks() -> tuple[dict, str]:
    """The roofline's denominators: MEASURED_PEAKS.json beside this file where it exists (its keys are looked
    for at any depth), else the fallback figures."""
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    found: dict = {}

    def walk(node) -> None:
        if isinstance(node, dict):
            for k, v in node.items():
                if k in FALLBACK_PEAKS and isinstance(v, (int, float)) and not isinstance(v, bool) and v > 0:
                    found.setdefault(k, float(v))
                else:
                    walk(v)
        elif isinstance(node, list):
            for v in node:
                walk(v)

    if os.path.isfile(path):
        try:
            with open(path) as fh:
                walk(json.load(fh))
        except (OSError, ValueError):
            found = {}
    if "hbm_gbs" in found and "bf16_tflops" in found:
        return {**FALLBACK_PEAKS, **found}, "measured"
    return dict(FALLBACK_PEAKS), "fallback"


def run_reference(args) -> int:
    from baseline.reference_arm import run
    return run(args)


def _free_device_memory() -> None:
    import gc

    import torch
    gc.collect()
    torch.cuda.empty_cache()


def run_ours(args) -> int:
    import torch

    from acvram_b200 import Engine, SamplingParams
    from acvram_b200 import bench as B
    from acvram_b200.config import Qwen3Config
    from acvram_b200.kernels import ops
    from acvram_b200.models import build_random

    t_begin = time.time()
    pk, pk_src = peaks()
    K, W = args.steps, args.warmup
    page = args.page_size
    refused: dict[str, str] = {}
    points: dict[str, float] = {}

    def build(shape_name: str, layers: int | None, max_batch: int, pool_tokens: int, max_model_len: int, budget: int = 4096):
        shape = SHAPES[shape_name]
        cfg = Qwen3Config(**{**shape, "num_hidden_layers": layers or shape["num_hidden_layers"]})
        t0 = time.time()
        model = build_random(cfg, seed=0, dtype=torch.bfloat16, device="cuda:0")
        torch.cuda.synchronize()
        print(f"[bench] {shape_name}: model built in {time.time() - t0:.1f} s ({model.weight_bytes() / 1e9:.2f} GB)",
              file=sys.stderr, flush=True)
        engine = Engine(model, "bfloat16", max_batch_size=max_batch, max_model_len=max_model_len, page_size=page,
                        num_pages=pool_tokens // page + 2 * max_batch + 8, token_budget=budget,
                        enable_cuda_graphs=not args.no_cuda_graphs,
                        enable_prefix_cache=False)     # every prompt is computed: no number rests on pages taken over
        return cfg, model, engine

    def decode_point(runner, batch: int, context: int, steps: int, warmup: int, sample_clocks: bool = False):
        names = [f"d{batch}-{context}-{i}" for i in range(batch)]
        B.fill_contexts(runner, names, context)
        torch.cuda.synchronize()
        try:
            if sample_clocks:
                with B.ClockSampler() as cs:
                    res = B.time_decode(runner, names, steps, warmup)
                res["clocks"] = cs.summary()
            else:
                res = B.time_decode(runner, names, steps, warmup)
        finally:
            for n in names:
                runner.release(n)
        mid = context + warmup + steps // 2
        res["bytes"] = B.decode_step_bytes(runner.model, batch, mid)
        res["gbs"] = res["bytes"] / (res["ms_per_step"] * 1e-3) / 1e9
        return res

    def point(name: str, fn) -> None:
        """One further point: its number, or why it was refused; never the end of the run."""
        try:
            fn()
        except B.Refused as exc:
            refused[name] = str(exc)
        except Exception as exc:  # noqa: BLE001  (a point beside the headline must not cost the headline)
            refused[name] = f"{type(exc).__name__}: {exc}"[:200]

    # ------------------------------------------------------------------ the headline shape
    shape = SHAPES[args.shape]
    full_layers = shape["num_hidden_layers"]
    layers = args.layers or full_layers
    fill_steps = -(-args.batch * args.context // 4096)        # steps in which the end-to-end run's prompts are computed
    per_request = args.context + 2 * (K + W) + fill_steps + 3 * page
    max_batch = max(args.batch, 64 if not args.skip_points else args.batch)
    long_ctx = 8192
    cfg, model, engine = build(args.shape, layers, max_batch, max_batch * per_request + 2048 + page, 8192)
    runner = engine.runner

    try:
        main = decode_point(runner, args.batch, args.context, K, W, sample_clocks=True)
    except B.Refused as exc:
        print(json.dumps({"metric": f"decode tok/s at batch {args.batch}", "value": None, "refused": str(exc), "n_gpus": 1,
                          "steps": K, "warmup": W}))
        return 3

    # end to end through the public entry point: host ids in, host ids out, every step
    def end_to_end(sp_of) -> tuple[float, int]:
        for i in range(args.batch):
            engine.add_request(B.synthetic_ids(cfg.vocab_size, args.context, 50 + i), sp_of(i))
        while any(r.remaining > 1 or r.computed == 0 for r in engine.scheduler.running) or engine.scheduler.waiting:
            engine.step()
        for _ in range(W):
            engine.step()
        torch.cuda.synchronize()
        replays0 = runner.graphs.replays if runner.graphs is not None else 0
        t0 = time.perf_counter()
        got = 0
        for _ in range(K):
            got += sum(len(o.token_ids) for o in engine.step())
        torch.cuda.synchronize()
        dt = time.perf_counter() - t0
        h2d = runner.builder.last_h2d_bytes
        replayed = (runner.graphs.replays - replays0) if runner.graphs is not None else K
        while not engine.idle:
            engine.step()
        if got != K * args.batch:
            raise B.Refused(f"{got} tokens came out of {K} steps of {args.batch} requests")
        if engine.stats.failed_steps:
            raise B.Refused(f"a step failed: {engine.last_error}")
        if runner.graphs is not None and runner.graphs.disabled_reason is None and replayed < K:
            raise B.Refused(f"{K - replayed} of {K} timed steps did not replay a captured graph")
        return got / dt, h2d

    # requests whose prompts are done decode while the others' prompts are computed: enough tokens for those steps too
    n_out = K + W + 4 + fill_steps
    graphs_on = bool(engine.enable_cuda_graphs)
    try:
        e2e_rate, h2d = end_to_end(lambda i: SamplingParams(temperature=0.0, max_tokens=n_out, ignore_eos=True))
        e2e = {"value": round(e2e_rate, 1), "unit": "tokens/s", "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": 4 * args.batch + 4}
    except B.Refused as exc:
        e2e = {"value": None, "unit": "tokens/s", "refused": str(exc)}
    # one prompt of 2048 tokens (a different one each time): 3 untimed, then the median of 5
    pre = B.time_prefill(runner, 2048, reps=5, warmup=3)
    pre_frac = B.prefill_flops(model, 2048) / (pre["ms"] * 1e-3) / (pk["bf16_tflops"] * 1e12)

    if not args.skip_points:
        for b in (1, 64):
            def f(b=b):
                r = decode_point(runner, b, args.context, K, W)
                points[f"decode_b{b}"] = round(r["tokens_per_s"], 1)
                points[f"decode_b{b}_hbm_frac"] = round(r["gbs"] / pk["hbm_gbs"], 4)
            point(f"decode_b{b}", f)

    if not args.skip_points:
        def sampled():
            rate, _ = end_to_end(lambda i: SamplingParams(temperature=0.7, top_p=0.9, max_tokens=n_out, ignore_eos=True, seed=i))
            points[f"sampled_b{args.batch}_e2e"] = round(rate, 1)
        point("sampled_e2e", sampled)

        def long_context():
            # contexts of 8192 tokens need room beyond the headline engine's 8192: a runner of its own on the same model
            from acvram_b200.engine.runner import ModelRunner
            nonlocal engine, runner
            del engine, runner
            _free_device_memory()
            tokens = args.batch * (long_ctx + 2 * (K + W) + 3 * page) + long_ctx + page
            long_runner = ModelRunner(model, page, tokens // page + 8, args.batch + 1, max_len=2 * long_ctx)
            if not args.no_cuda_graphs:
                long_runner.enable_graphs()
            r = decode_point(long_runner, args.batch, long_ctx, K, W)
            points[f"decode_b{args.batch}_ctx{long_ctx}"] = round(r["tokens_per_s"], 1)
            points[f"decode_b{args.batch}_ctx{long_ctx}_hbm_frac"] = round(r["gbs"] / pk["hbm_gbs"], 4)
            p8 = B.time_prefill(long_runner, long_ctx, reps=3, warmup=1)
            points[f"prefill_{long_ctx}"] = round(p8["tokens_per_s"], 1)
            points[f"prefill_{long_ctx}_frac"] = round(B.prefill_flops(model, long_ctx) / (p8["ms"] * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)
        point("long_context", long_context)

    line = {
        "metric": f"decode tok/s at batch {args.batch} (Qwen3-{args.shape.upper()} shape, {args.context}-token contexts)",
        "value": round(main["tokens_per_s"], 1), "unit": "tokens/s", "n_gpus": 1, "steps": K, "warmup": W,
        "ms_per_step": round(main["ms_per_step"], 4), "higher_is_better": True, "scaling": "weak",
        "vs_baseline": None, "dtype": "bf16", "data": "synthetic token ids, random weights N(0,0.02)",
        "config": bench_config(args, cfg.to_dict(), layers, full_layers, page, graphs_on),
        "clocks": main.get("clocks"),
        "e2e": e2e,
        "gpu_launches": main["launches"],
        "prefill": {"value": round(pre["tokens_per_s"], 1), "tokens": 2048, "ms": round(pre["ms"], 3),
                    "frac": round(pre_frac, 4), "peak_tflops": pk["bf16_tflops"], "peaks": pk_src,
                    # the same against what cuBLAS holds back to back for seconds under the power cap: a prompt's
                    # step is 26 ms of dense products, run eight times in a row here
                    "frac_of_sustained": round(pre_frac * pk["bf16_tflops"] / pk["bf16_tflops_sustained"], 4)},
        "roofline": {"bound": "hbm", "achieved": round(main["gbs"], 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(main["gbs"] / pk["hbm_gbs"], 4), "peaks": pk_src},
        "points": points,
    }

    # ------------------------------------------------------------------ the other shapes that the baseline names
    if not args.skip_points and args.shape == "8b" and not args.layers:
        engine = runner = model = None
        _free_device_memory()

        def shape_14b():
            # a step of serving under load: 32 requests decode beside a 1024-token portion of another's prompt
            _, model14, eng14 = build("14b", None, 40, 33 * (2048 + 2 * (K + W) + 64) + 4096, 8192)
            try:
                names = [f"m{i}" for i in range(32)]
                B.fill_contexts(eng14.runner, names, 2048)
                r = B.time_mixed(eng14.runner, names, 1024, 2048, K, W)
                cost = model14.step_cost([1] * 32 + [1024], [2048 + W + K // 2] * 32 + [1536], 33)
                points["mixed_14b_32dec_1024_ms"] = round(r["ms_per_step"], 3)
                points["mixed_14b_32dec_1024_tok_s"] = round(r["tokens_per_s"], 1)
                points["mixed_14b_tflops_frac"] = round(cost["flops"] / (r["ms_per_step"] * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)
            finally:
                del eng14, model14
                _free_device_memory()
        if time.time() - t_begin < args.time_limit:
            point("mixed_14b", shape_14b)
        else:
            refused["mixed_14b"] = "left out: the run's time limit was reached"

        def shape_32b():
            _, model32, eng32 = build("32b", None, 64, 64 * (2048 + 2 * (K + W) + 64) + 4096, 16384)
            try:
                for b in (1, 8, 64):
                    r = decode_point(eng32.runner, b, 2048, K, W)
                    points[f"decode_32b_b{b}"] = round(r["tokens_per_s"], 1)
                    points[f"decode_32b_b{b}_hbm_frac"] = round(r["gbs"] / pk["hbm_gbs"], 4)
                p32 = B.time_prefill(eng32.runner, 2048, reps=3, warmup=1)
                points["prefill_32b_2048"] = round(p32["tokens_per_s"], 1)
                points["prefill_32b_2048_frac"] = round(B.prefill_flops(model32, 2048) / (p32["ms"] * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)
            finally:
                del eng32, model32
                _free_device_memory()
        if time.time() - t_begin < args.time_limit:
            point("shape_32b", shape_32b)
        else:
            refused["shape_32b"] = "left out: the run's time limit was reached"

    if refused:
        line["refused"] = refused
    print(json.dumps(line))
    return 0


# ---------------------------------------------------------------------- another design beside its closest relative
ZOTONEX_SIZES = {
    # width, heads, kv heads, dim (a head has two query vectors of it), vdim, chunk, experts, top, expert ff, shared ff
    "s": dict(width=2048, heads=16, kv_heads=4, dim=64, vdim=128, chunk=1024, experts=32, top=4, ff=512, shared_ff=1024),
    "m": dict(width=4096, heads=32, kv_heads=8, dim=64, vdim=128, chunk=2048, experts=64, top=6, ff=768, shared_ff=1536),
}


REDUDRA_SIZES = {
    # width; attention: heads, kv heads, head size (keys and values), window, kept first tokens; retention: heads, key size,
    # value size; recurrence: channels, blocks, taps; feed-forward size
    "s": dict(width=2048, heads=16, kv_heads=4, dim=128, window=1024, keep=8, r_heads=8, r_dim=64, r_vdim=128,
              channels=2048, blocks=16, taps=4, ff=6144),
    "m": dict(width=4096, heads=32, kv_heads=8, dim=128, window=2048, keep=8, r_heads=16, r_dim=64, r_vdim=128,
              channels=4096, blocks=16, taps=4, ff=12288),
}

NIZEDRA_SIZES = {
    # width; attention: heads, kv heads, head size (keys and values), where the distance-bias table ends (32 rows);
    # lightning: heads, key size, value size; latent attention: heads, unrotated and rotated key size, value size, ranks
    # of the query and key/value latents, window; feed-forward size (two matrices: 3/2 of the gated relative's three)
    "s": dict(width=2048, heads=16, kv_heads=4, dim=128, bias_max=4096, l_heads=16, l_dim=128, l_vdim=128,
              m_heads=16, m_dim=64, m_rot=64, m_vdim=128, q_rank=768, kv_rank=512, window=1024, ff=9216),
    "m": dict(width=4096, heads=32, kv_heads=8, dim=128, bias_max=4096, l_heads=32, l_dim=128, l_vdim=128,
              m_heads=32, m_dim=64, m_rot=64, m_vdim=128, q_rank=1536, kv_rank=512, window=2048, ff=18432),
}


VADELIX_SIZES = {
    # width, norm groups, taps; attention (both kinds): heads, kv heads, head size (keys and values), rotated part, window of
    # the windowed kind; time mixing: heads, head size; gated feed-forward size; mixture: experts, choices, groups, kept
    # groups, an expert's size, the shared expert's
    "s": dict(width=2048, groups=8, taps=4, heads=16, kv_heads=4, dim=128, rot=64, window=1024, t_heads=32, t_dim=64, ff=6144,
              experts=32, top=4, e_groups=8, e_keep=4, e_ff=768, shared_ff=1536),
    "m": dict(width=4096, groups=8, taps=4, heads=32, kv_heads=8, dim=128, rot=64, window=2048, t_heads=64, t_dim=64, ff=12288,
              experts=64, top=6, e_groups=8, e_keep=4, e_ff=1024, shared_ff=2048),
}


LODALIX_SIZES = {
    # width; latent attention (both kinds): heads, unrotated and rotated key size, value size, ranks of the query and key/value
    # latents; recurrence: heads, head size; gated feed-forward size
    "s": dict(width=2048, heads=16, dim=64, rot=64, vdim=128, q_rank=768, kv_rank=512, t_heads=32, t_dim=64, ff=6144),
    "m": dict(width=4096, heads=32, dim=64, rot=64, vdim=128, q_rank=1536, kv_rank=512, t_heads=64, t_dim=64, ff=12288),
}


def run_lodalix(args) -> int:
    """``--design lodalix``: prefill and decode throughput of the Lodalix design at layer sizes of real models (random
    weights; six layers: gated latent attention, latent attention with sinks, delta recurrence, gated latent attention on the
    first layer's rows, latent attention, recurrence), beside the closest models of the framework at equal size: a Nizedra
    model with latent attention of the same sizes and no window, and its other recurrence, in the same order of layers; and
    a Vadelix model's time mixing and gated unit.  Whole steps through the step function, and the mixer and feed-forward
    of each kind of layer alone with their rooflines (L2 flushed before each timed run).  One JSON line."""
    import torch

    from acvram_b200 import bench as B
    from acvram_b200.config import LodalixConfig, NizedraConfig, VadelixConfig
    from acvram_b200.engine.runner import ModelRunner
    from acvram_b200.models import build_random

    pk, pk_src = peaks()
    K, W = args.steps, args.warmup
    page = 64
    layers, vocab = args.layers or 6, 32768
    out = {"design": "lodalix", "beside": ["nizedra", "vadelix"], "layers": layers, "vocab": vocab, "dtype": "bf16",
           "page_size": page, "data": "synthetic token ids, random weights", "peaks": {**pk, "source": pk_src}, "sizes": {}}
    for name in args.sizes.split(","):
        z = LODALIX_SIZES[name]
        rows = {"heads": z["heads"], "dim": z["dim"], "rot_dim": z["rot"], "vdim": z["vdim"], "q_rank": z["q_rank"],
                "kv_rank": z["kv_rank"], "scale": (z["dim"] + z["rot"]) ** -0.5, "rot": {"base": 1e6, "dims": z["rot"]}}
        gated = {**rows, "rot": {**rows["rot"], "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
        head = {"heads": z["t_heads"], "dim": z["t_dim"]}
        order = (("latent_attention_2", gated), ("latent_attention", rows), ("general_delta", head),
                 ("latent_attention_2", {**gated, "kv_from": 0}), ("latent_attention", rows), ("general_delta", head))
        unit = {"kind": "dense", "ff": z["ff"], "limit": 7.0}
        lcfg = LodalixConfig.from_dict({"architecture": "Lodalix", "vocab": vocab, "width": z["width"], "norm": {"eps": 1e-6},
                                        "layers": [{"type": order[i % 6][0], "mixer": order[i % 6][1], "mlp": unit} for i in range(layers)]})
        light = {"heads": z["heads"], "dim": z["vdim"], "vdim": z["vdim"], "decay": [1.0 - 2.0 ** (-4 - i % 8) for i in range(z["heads"])]}
        ncfg = NizedraConfig.from_dict({
            "architecture": "Nizedra", "vocab": vocab, "width": z["width"], "norm": {"eps": 1e-6},
            "layers": [{"type": "lightning", "mixer": light, "mlp": {"kind": "dense", "ff": z["ff"] * 3 // 2}} if i % 3 == 2 else
                       {"type": "latent_attention", "mixer": rows, "mlp": {"kind": "dense", "ff": z["ff"] * 3 // 2}} for i in range(layers)]})
        vcfg = VadelixConfig.from_dict({
            "architecture": "Vadelix", "vocab": vocab, "width": z["width"], "norm": {"eps": 1e-6, "groups": 1}, "residual_mult": 1.0,
            "canon": {"taps": 1}, "layers": [{"type": "wkv", "mixer": head, "mlp": {"kind": "dense", "ff": z["ff"]}}]})
        kinds_of = {"lodalix": (("gated_latent", 0), ("sink_latent", 1), ("delta", 2), ("borrowed_latent", 3)),
                    "nizedra": (("latent", 0), ("lightning", 2)), "vadelix": (("wkv", 0),)}
        res = {"sizes": dict(z)}
        for arm, cfg in (("lodalix", lcfg), ("nizedra", ncfg), ("vadelix", vcfg)):
            model = build_random(cfg, seed=0, dtype=torch.bfloat16, device="cuda:0")
            batch_max = 64
            tokens = batch_max * (args.context + 2 * (K + W) + 2 * page) + 4096
            runner = ModelRunner(model, page, tokens // page + 8, batch_max + 2, max_len=8192)
            if not args.no_cuda_graphs:
                runner.enable_graphs()
            r = {"weights_gb": round(model.weight_bytes() / 1e9, 3)}
            try:
                if arm != "vadelix":
                    pre = B.time_prefill(runner, 2048, reps=5, warmup=3)
                    flops = B.prefill_flops(model, 2048)
                    r["prefill_2048"] = {"tokens_per_s": round(pre["tokens_per_s"], 1), "ms": round(pre["ms"], 3),
                                         "tflops_frac": round(flops / (pre["ms"] * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)}
                    for b in (8, 64):
                        names = [f"d{b}-{i}" for i in range(b)]
                        B.fill_contexts(runner, names, args.context)
                        try:
                            d = B.time_decode(runner, names, K, W)
                        finally:
                            for n in names:
                                runner.release(n)
                        nbytes = B.decode_step_bytes(model, b, args.context + W + K // 2)
                        r[f"decode_b{b}"] = {"tokens_per_s": round(d["tokens_per_s"], 1), "ms_per_step": round(d["ms_per_step"], 4),
                                             "hbm_frac": round(nbytes / (d["ms_per_step"] * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}
                for kind, layer in kinds_of[arm]:
                    if layer >= layers:
                        continue
                    for label, ql, kl in (("prefill_2048", [2048], [2048]), ("decode_b64", [1] * 64, [args.context] * 64)):
                        for part, v in B.time_parts(runner, ql, kl, layer=layer).items():
                            if part == "feed_forward" and layer:
                                continue        # (the same in every layer)
                            sec = v["ms"] * 1e-3
                            r[f"{kind if part == 'mixer' else 'feed_forward'}_{label}"] = {
                                "us": round(v["ms"] * 1e3, 1),
                                "tflops_frac": round(v["flops"] / sec / (pk["bf16_tflops"] * 1e12), 4),
                                "hbm_frac": round(v["bytes"] / sec / 1e9 / pk["hbm_gbs"], 4)}
            except B.Refused as exc:
                r["refused"] = str(exc)
            res[arm + "_result"] = r
            del runner, model
            _free_device_memory()
        out["sizes"][name] = res
    print(json.dumps(out))
    return 0


ZOGAPEL_SIZES = {
    # width; attention: heads, kv heads, head size, rotated part, window; recurrence: value heads, query/key heads, key size,
    # value size, taps; dense feed-forward size (two matrices); mixture: experts, choices, an expert's size
    "s": dict(width=2048, heads=16, kv_heads=4, dim=128, rot=64, window=1024, d_heads=16, d_kv=8, d_dim=128, d_vdim=128, taps=4,
              ff=9216, experts=32, top=4, e_ff=768),
    "m": dict(width=4096, heads=32, kv_heads=8, dim=128, rot=64, window=2048, d_heads=32, d_kv=16, d_dim=128, d_vdim=128, taps=4,
              ff=18432, experts=64, top=6, e_ff=1024),
}


def run_zogapel(args) -> int:
    """``--design zogapel``: prefill and decode throughput of the Zogapel design at layer sizes of real models (random
    weights; six layers: windowed attention whose values are its keys and the gated delta rule in turn, a dense feed-forward
    in every third layer and a mixture in the others), beside the closest models of the framework at equal size: a Vadelix
    model with windowed attention of the same heads, its own recurrence with as much state, and feed-forwards of equal weight
    count; one layer of Lodalix for the delta rule (as many heads of the same size); one of Nizedra for the dense unit.
    Whole steps through the step function, and the mixer and feed-forward of each kind of layer alone with their
    rooflines (L2 flushed before each timed run).  One JSON line."""
    import torch

    from acvram_b200 import bench as B
    from acvram_b200.config import LodalixConfig, NizedraConfig, VadelixConfig, ZogapelConfig
    from acvram_b200.engine.runner import ModelRunner
    from acvram_b200.models import build_random

    pk, pk_src = peaks()
    K, W = args.steps, args.warmup
    page = 64
    layers, vocab = args.layers or 6, 32768
    out = {"design": "zogapel", "beside": ["vadelix", "lodalix", "nizedra"], "layers": layers, "vocab": vocab, "dtype": "bf16",
           "page_size": page, "data": "synthetic token ids, random weights", "peaks": {**pk, "source": pk_src}, "sizes": {}}
    for name in args.sizes.split(","):
        z = ZOGAPEL_SIZES[name]
        heads = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"], "scale": z["dim"] ** -0.5,
                 "mask": {"size": z["window"]}}
        rot = {"base": 1e6, "dims": z["rot"], "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}
        gated = {"heads": z["d_heads"], "kv_heads": z["d_kv"], "dim": z["d_dim"], "vdim": z["d_vdim"], "conv": z["taps"]}
        dense, moe = {"kind": "dense", "ff": z["ff"]}, {"kind": "moe", "router": {"experts": z["experts"], "top": z["top"]}, "expert": {"ff": z["e_ff"]}}
        zcfg = ZogapelConfig.from_dict({
            "architecture": "Zogapel", "vocab": vocab, "width": z["width"], "embedding": {"scale": 1.0}, "norm": {"eps": 1e-6},
            "layers": [{"type": "delta", "mixer": gated, "mlp": moe if i % 3 else dense} if i % 2 else
                       {"type": "attention", "mixer": {**heads, "rot": rot}, "mlp": moe if i % 3 else dense} for i in range(layers)]})
        # (a gated unit has three matrices, a plain expert two; the relative's mixture always has a shared expert: a small one)
        v_dense = {"kind": "dense", "ff": z["ff"] * 2 // 3}
        v_moe = {"kind": "moe", "expert": {"ff": z["e_ff"] * 3 // 2}, "shared": {"ff": 64},
                 "router": {"experts": z["experts"], "top": z["top"], "groups": {"count": 1, "keep": 1}}}
        v_mixer = {**heads, "v_mix": False, "q_temp": {"coef": 0.1, "every": 512}}
        state = z["d_heads"] * z["d_dim"] * z["d_vdim"]
        wkv = {"heads": state // (64 * 64), "dim": 64}
        vcfg = VadelixConfig.from_dict({
            "architecture": "Vadelix", "vocab": vocab, "width": z["width"], "norm": {"eps": 1e-6, "groups": 1}, "residual_mult": 1.0,
            "canon": {"taps": 1},
            "layers": [{"type": "wkv", "mixer": wkv, "mlp": v_moe if i % 3 else v_dense} if i % 2 else
                       {"type": "attention_2", "mixer": v_mixer, "mlp": v_moe if i % 3 else v_dense} for i in range(layers)]})
        lcfg = LodalixConfig.from_dict({
            "architecture": "Lodalix", "vocab": vocab, "width": z["width"], "norm": {"eps": 1e-6},
            "layers": [{"type": "general_delta", "mixer": {"heads": z["d_heads"], "dim": z["d_dim"]}, "mlp": None}]})
        light = {"heads": z["d_heads"], "dim": z["d_dim"], "vdim": z["d_vdim"], "decay": [1.0 - 2.0 ** (-4 - i % 8) for i in range(z["d_heads"])]}
        ncfg = NizedraConfig.from_dict({"architecture": "Nizedra", "vocab": vocab, "width": z["width"], "norm": {"eps": 1e-6},
                                        "layers": [{"type": "lightning", "mixer": light, "mlp": dense}]})
        kinds_of = {"zogapel": (("attention", 0, "dense"), ("gated_delta", 1, "moe")),
                    "vadelix": (("attention", 0, "gated_unit"), ("wkv", 1, "moe")),
                    "lodalix": (("general_delta", 0, None),), "nizedra": (("lightning", 0, "dense"),)}
        res = {"sizes": dict(z)}
        for arm, cfg in (("zogapel", zcfg), ("vadelix", vcfg), ("lodalix", lcfg), ("nizedra", ncfg)):
            model = build_random(cfg, seed=0, dtype=torch.bfloat16, device="cuda:0")
            batch_max = 64
            tokens = batch_max * (args.context + 2 * (K + W) + 2 * page) + 4096
            runner = ModelRunner(model, page, tokens // page + 8, batch_max + 2, max_len=8192)
            if not args.no_cuda_graphs:
                runner.enable_graphs()
            r = {"weights_gb": round(model.weight_bytes() / 1e9, 3)}
            try:
                if arm in ("zogapel", "vadelix"):
                    pre = B.time_prefill(runner, 2048, reps=5, warmup=3)
                    flops = B.prefill_flops(model, 2048)
                    r["prefill_2048"] = {"tokens_per_s": round(pre["tokens_per_s"], 1), "ms": round(pre["ms"], 3),
                                         "tflops_frac": round(flops / (pre["ms"] * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)}
                    for b in (8, 64):
                        names = [f"d{b}-{i}" for i in range(b)]
                        B.fill_contexts(runner, names, args.context)
                        try:
                            d = B.time_decode(runner, names, K, W)
                        finally:
                            for n in names:
                                runner.release(n)
                        nbytes = B.decode_step_bytes(model, b, args.context + W + K // 2)
                        r[f"decode_b{b}"] = {"tokens_per_s": round(d["tokens_per_s"], 1), "ms_per_step": round(d["ms_per_step"], 4),
                                             "hbm_frac": round(nbytes / (d["ms_per_step"] * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}
                for kind, layer, unit in kinds_of[arm]:
                    if layer >= layers:
                        continue
                    for label, ql, kl in (("prefill_2048", [2048], [2048]), ("decode_b64", [1] * 64, [args.context] * 64)):
                        for part, v in B.time_parts(runner, ql, kl, layer=layer).items():
                            what = kind if part == "mixer" else unit
                            if what is None:
                                continue
                            sec = v["ms"] * 1e-3
                            r[f"{what}_{label}"] = {"us": round(v["ms"] * 1e3, 1),
                                                    "tflops_frac": round(v["flops"] / sec / (pk["bf16_tflops"] * 1e12), 4),
                                                    "hbm_frac": round(v["bytes"] / sec / 1e9 / pk["hbm_gbs"], 4)}
            except B.Refused as exc:
                r["refused"] = str(exc)
            res[arm + "_result"] = r
            del runner, model
            _free_device_memory()
        out["sizes"][name] = res
    print(json.dumps(out))
    return 0


def run_vadelix(args) -> int:
    """``--design vadelix``: prefill and decode throughput of the Vadelix design at layer sizes of real models (random
    weights; six layers: time mixing, rotated attention with sinks, windowed attention with slopes, twice, gated
    feed-forwards and mixtures in turn), beside a Qwen3 model of equal size: the same width, as many attention heads of
    the same size, the gated feed-forward's size.  Whole steps through the step function, and the mixer and feed-forward
    of each kind of layer alone with their rooflines (L2 flushed before each timed run).  One JSON line."""
    import torch

    from acvram_b200 import bench as B
    from acvram_b200.config import Qwen3Config, VadelixConfig
    from acvram_b200.engine.runner import ModelRunner
    from acvram_b200.models import build_random

    pk, pk_src = peaks()
    K, W = args.steps, args.warmup
    page = 64
    layers, vocab = args.layers or 6, 32768
    out = {"design": "vadelix", "beside": "qwen3", "layers": layers, "vocab": vocab, "dtype": "bf16", "page_size": page,
           "data": "synthetic token ids, random weights", "peaks": {**pk, "source": pk_src}, "sizes": {}}
    for name in args.sizes.split(","):
        z = VADELIX_SIZES[name]
        dense = {"kind": "dense", "ff": z["ff"]}
        moe = {"kind": "moe", "expert": {"ff": z["e_ff"]}, "shared": {"ff": z["shared_ff"]},
               "router": {"experts": z["experts"], "top": z["top"], "groups": {"count": z["e_groups"], "keep": z["e_keep"]}}}
        heads = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"], "scale": z["dim"] ** -0.5,
                 "v_mix": True}
        mixers = (("wkv", {"heads": z["t_heads"], "dim": z["t_dim"]}),
                  ("attention", {**heads, "rot": {"base": 1e6, "dims": z["rot"],
                                                  "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}),
                  ("attention_2", {**heads, "mask": {"size": z["window"]}, "q_temp": {"coef": 0.1, "every": 512}}))
        vcfg = VadelixConfig.from_dict({
            "architecture": "Vadelix", "vocab": vocab, "width": z["width"], "norm": {"eps": 1e-6, "groups": z["groups"]},
            "residual_mult": 0.5, "canon": {"taps": z["taps"]},
            "layers": [{"type": mixers[i % 3][0], "mixer": mixers[i % 3][1], "mlp": moe if i % 2 else dense} for i in range(layers)]})
        qcfg = Qwen3Config(vocab_size=vocab, hidden_size=z["width"], intermediate_size=z["ff"], num_hidden_layers=layers,
                           num_attention_heads=z["heads"], num_key_value_heads=z["kv_heads"], head_dim=z["dim"],
                           rms_norm_eps=1e-6, rope_theta=1e6, max_position_embeddings=8192, tie_word_embeddings=False)
        res = {"vadelix": dict(z), "qwen3": {"hidden": qcfg.hidden_size, "intermediate": qcfg.intermediate_size,
                                            "q_heads": qcfg.num_attention_heads, "kv_heads": qcfg.num_key_value_heads,
                                            "head_dim": qcfg.head_dim}}
        for arm, cfg in (("vadelix", vcfg), ("qwen3", qcfg)):
            model = build_random(cfg, seed=0, dtype=torch.bfloat16, device="cuda:0")
            batch_max = 64
            tokens = batch_max * (args.context + 2 * (K + W) + 2 * page) + 4096
            runner = ModelRunner(model, page, tokens // page + 8, batch_max + 2, max_len=8192)
            if not args.no_cuda_graphs:
                runner.enable_graphs()
            r = {"weights_gb": round(model.weight_bytes() / 1e9, 3)}
            try:
                pre = B.time_prefill(runner, 2048, reps=5, warmup=3)
                flops = B.prefill_flops(model, 2048)
                r["prefill_2048"] = {"tokens_per_s": round(pre["tokens_per_s"], 1), "ms": round(pre["ms"], 3),
                                     "tflops_frac": round(flops / (pre["ms"] * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)}
                for b in (8, 64):
                    names = [f"d{b}-{i}" for i in range(b)]
                    B.fill_contexts(runner, names, args.context)
                    try:
                        d = B.time_decode(runner, names, K, W)
                    finally:
                        for n in names:
                            runner.release(n)
                    nbytes = B.decode_step_bytes(model, b, args.context + W + K // 2)
                    r[f"decode_b{b}"] = {"tokens_per_s": round(d["tokens_per_s"], 1), "ms_per_step": round(d["ms_per_step"], 4),
                                         "hbm_frac": round(nbytes / (d["ms_per_step"] * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}
                # layer 0: time mixing + gated unit; 1: rotated attention + mixture; 2: windowed attention
                kinds = (("wkv", 0), ("attention", 1), ("window", 2)) if arm == "vadelix" and layers > 2 else (("", 0),)
                for kind, layer in kinds:
                    for label, ql, kl in (("prefill_2048", [2048], [2048]), ("decode_b64", [1] * 64, [args.context] * 64)):
                        parts = B.time_parts(runner, ql, kl, layer=layer)
                        for part, v in parts.items():
                            if part == "feed_forward" and layer > 1:
                                continue        # the feed-forwards of layers 0 and 1 are the two kinds
                            sec = v["ms"] * 1e-3
                            label_part = ("gated_unit" if layer == 0 else "mixture") if part == "feed_forward" and kind else part
                            r[f"{kind + '_' if kind and part == 'mixer' else ''}{label_part}_{label}"] = {
                                "us": round(v["ms"] * 1e3, 1),
                                "tflops_frac": round(v["flops"] / sec / (pk["bf16_tflops"] * 1e12), 4),
                                "hbm_frac": round(v["bytes"] / sec / 1e9 / pk["hbm_gbs"], 4)}
            except B.Refused as exc:
                r["refused"] = str(exc)
            res[arm + "_result"] = r
            del runner, model
            _free_device_memory()
        out["sizes"][name] = res
    print(json.dumps(out))
    return 0


def run_nizedra(args) -> int:
    """``--design nizedra``: prefill and decode throughput of the Nizedra design at layer sizes of real models (random
    weights; six layers: mixed-heads attention, lightning, latent attention, twice), beside a Qwen3 model of equal size:
    the same width, as many attention heads of the same size, a gated feed-forward with as many weights.  Whole steps
    through the step function, and the mixer and feed-forward of each kind of layer alone with their rooflines (L2
    flushed before each timed run).  One JSON line."""
    import torch

    from acvram_b200 import bench as B
    from acvram_b200.config import NizedraConfig, Qwen3Config
    from acvram_b200.engine.runner import ModelRunner
    from acvram_b200.models import build_random

    pk, pk_src = peaks()
    K, W = args.steps, args.warmup
    page = 64
    layers, vocab = args.layers or 6, 32768
    out = {"design": "nizedra", "beside": "qwen3", "layers": layers, "vocab": vocab, "dtype": "bf16", "page_size": page,
           "data": "synthetic token ids, random weights", "peaks": {**pk, "source": pk_src}, "sizes": {}}
    for name in args.sizes.split(","):
        z = NIZEDRA_SIZES[name]
        mlp = {"kind": "dense", "ff": z["ff"]}
        att = {"type": "attention", "mlp": mlp, "mixer": {
            "heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"], "scale": z["dim"] ** -0.5 * 8.0,
            "softcap": 50.0, "bias_max": z["bias_max"]}}
        lig = {"type": "lightning", "mlp": mlp, "mixer": {
            "heads": z["l_heads"], "dim": z["l_dim"], "vdim": z["l_vdim"],
            "decay": [1.0 - 2.0 ** (-5 - 3 * h / z["l_heads"]) for h in range(z["l_heads"])]}}
        lat = {"type": "latent_attention", "mlp": mlp, "mixer": {
            "heads": z["m_heads"], "dim": z["m_dim"], "rot_dim": z["m_rot"], "vdim": z["m_vdim"], "q_rank": z["q_rank"],
            "kv_rank": z["kv_rank"], "scale": (z["m_dim"] + z["m_rot"]) ** -0.5, "mask": {"size": z["window"]},
            "rot": {"base": 1e6, "dims": z["m_rot"]}}}
        kinds3 = (att, lig, lat)
        ncfg = NizedraConfig.from_dict({"architecture": "Nizedra", "vocab": vocab, "width": z["width"], "norm": {"eps": 1e-6},
                                        "layers": [kinds3[i % 3] for i in range(layers)]})
        qcfg = Qwen3Config(vocab_size=vocab, hidden_size=z["width"], intermediate_size=z["ff"] * 2 // 3, num_hidden_layers=layers,
                           num_attention_heads=z["heads"], num_key_value_heads=z["kv_heads"], head_dim=z["dim"],
                           rms_norm_eps=1e-6, rope_theta=1e6, max_position_embeddings=8192, tie_word_embeddings=False)
        res = {"nizedra": dict(z), "qwen3": {"hidden": qcfg.hidden_size, "intermediate": qcfg.intermediate_size,
                                            "q_heads": qcfg.num_attention_heads, "kv_heads": qcfg.num_key_value_heads,
                                            "head_dim": qcfg.head_dim}}
        for arm, cfg in (("nizedra", ncfg), ("qwen3", qcfg)):
            model = build_random(cfg, seed=0, dtype=torch.bfloat16, device="cuda:0")
            batch_max = 64
            tokens = batch_max * (args.context + 2 * (K + W) + 2 * page) + 4096
            runner = ModelRunner(model, page, tokens // page + 8, batch_max + 2, max_len=8192)
            if not args.no_cuda_graphs:
                runner.enable_graphs()
            r = {"weights_gb": round(model.weight_bytes() / 1e9, 3)}
            try:
                pre = B.time_prefill(runner, 2048, reps=5, warmup=3)
                flops = B.prefill_flops(model, 2048)
                r["prefill_2048"] = {"tokens_per_s": round(pre["tokens_per_s"], 1), "ms": round(pre["ms"], 3),
                                     "tflops_frac": round(flops / (pre["ms"] * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)}
                for b in (8, 64):
                    names = [f"d{b}-{i}" for i in range(b)]
                    B.fill_contexts(runner, names, args.context)
                    try:
                        d = B.time_decode(runner, names, K, W)
                    finally:
                        for n in names:
                            runner.release(n)
                    nbytes = B.decode_step_bytes(model, b, args.context + W + K // 2)
                    r[f"decode_b{b}"] = {"tokens_per_s": round(d["tokens_per_s"], 1), "ms_per_step": round(d["ms_per_step"], 4),
                                         "hbm_frac": round(nbytes / (d["ms_per_step"] * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}
                kinds = (("attention", 0), ("lightning", 1), ("latent", 2)) if arm == "nizedra" and layers > 2 else (("", 0),)
                for kind, layer in kinds:
                    for label, ql, kl in (("prefill_2048", [2048], [2048]), ("decode_b64", [1] * 64, [args.context] * 64)):
                        parts = B.time_parts(runner, ql, kl, layer=layer)
                        for part, v in parts.items():
                            if part == "feed_forward" and layer:
                                continue        # every layer's feed-forward is the same
                            sec = v["ms"] * 1e-3
                            r[f"{kind + '_' if kind else ''}{part}_{label}"] = {
                                "us": round(v["ms"] * 1e3, 1),
                                "tflops_frac": round(v["flops"] / sec / (pk["bf16_tflops"] * 1e12), 4),
                                "hbm_frac": round(v["bytes"] / sec / 1e9 / pk["hbm_gbs"], 4)}
            except B.Refused as exc:
                r["refused"] = str(exc)
            res[arm + "_result"] = r
            del runner, model
            _free_device_memory()
        out["sizes"][name] = res
    print(json.dumps(out))
    return 0


def run_redudra(args) -> int:
    """``--design redudra``: prefill and decode throughput of the Redudra design at layer sizes of real models (random
    weights; four layers, parallel and recurrent ones in turn), beside a Qwen3 model of equal size: the same width, as
    many attention heads of the same size, the same feed-forward size.  Whole steps through the step function, and the
    mixer and feed-forward of a parallel layer and of a recurrent layer alone with their rooflines (L2 flushed before
    each timed run).  One JSON line."""
    import torch

    from acvram_b200 import bench as B
    from acvram_b200.config import Qwen3Config, RedudraConfig
    from acvram_b200.engine.runner import ModelRunner
    from acvram_b200.models import build_random

    pk, pk_src = peaks()
    K, W = args.steps, args.warmup
    page = 64
    layers, vocab = args.layers or 4, 32768
    out = {"design": "redudra", "beside": "qwen3", "layers": layers, "vocab": vocab, "dtype": "bf16", "page_size": page,
           "data": "synthetic token ids, random weights", "peaks": {**pk, "source": pk_src}, "sizes": {}}
    for name in args.sizes.split(","):
        z = REDUDRA_SIZES[name]
        par = {"type": "parallel", "mlp": {"kind": "dense", "ff": z["ff"]}, "mixer": {
            "left": {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"], "scale": z["dim"] ** -0.5,
                     "mask": {"size": z["window"], "keep_first": z["keep"]},
                     "rot": {"base": 1e6, "dims": z["dim"], "scaling": {"factor": 8.0, "original": 4096, "fast": 16.0, "slow": 2.0}}},
            "right": {"heads": z["r_heads"], "dim": z["r_dim"], "vdim": z["r_vdim"],
                      "decay": [1.0 - 2.0 ** (-5 - 3 * h / z["r_heads"]) for h in range(z["r_heads"])],
                      "rot": {"base": 1e4, "dims": z["r_dim"]}},
            "left_scale": 0.7, "right_scale": 0.4}}
        rec = {"type": "rglru", "mlp": {"kind": "dense", "ff": z["ff"]},
               "mixer": {"width": z["channels"], "blocks": z["blocks"], "conv": z["taps"]}}
        rcfg = RedudraConfig.from_dict({"architecture": "Redudra", "vocab": vocab, "width": z["width"], "norm": {"eps": 1e-6},
                                        "residual_mult": 0.4, "logit_softcap": 50.0,
                                        "layers": [par if i % 2 == 0 else rec for i in range(layers)]})
        qcfg = Qwen3Config(vocab_size=vocab, hidden_size=z["width"], intermediate_size=z["ff"], num_hidden_layers=layers,
                           num_attention_heads=z["heads"], num_key_value_heads=z["kv_heads"], head_dim=z["dim"],
                           rms_norm_eps=1e-6, rope_theta=1e6, max_position_embeddings=8192, tie_word_embeddings=False)
        res = {"redudra": dict(z), "qwen3": {"hidden": qcfg.hidden_size, "intermediate": qcfg.intermediate_size,
                                            "q_heads": qcfg.num_attention_heads, "kv_heads": qcfg.num_key_value_heads,
                                            "head_dim": qcfg.head_dim}}
        for arm, cfg in (("redudra", rcfg), ("qwen3", qcfg)):
            model = build_random(cfg, seed=0, dtype=torch.bfloat16, device="cuda:0")
            batch_max = 64
            tokens = batch_max * (args.context + 2 * (K + W) + 2 * page) + 4096
            runner = ModelRunner(model, page, tokens // page + 8, batch_max + 2, max_len=8192)
            if not args.no_cuda_graphs:
                runner.enable_graphs()
            r = {"weights_gb": round(model.weight_bytes() / 1e9, 3)}
            try:
                pre = B.time_prefill(runner, 2048, reps=5, warmup=3)
                flops = B.prefill_flops(model, 2048)
                r["prefill_2048"] = {"tokens_per_s": round(pre["tokens_per_s"], 1), "ms": round(pre["ms"], 3),
                                     "tflops_frac": round(flops / (pre["ms"] * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)}
                for b in (8, 64):
                    names = [f"d{b}-{i}" for i in range(b)]
                    B.fill_contexts(runner, names, args.context)
                    try:
                        d = B.time_decode(runner, names, K, W)
                    finally:
                        for n in names:
                            runner.release(n)
                    nbytes = B.decode_step_bytes(model, b, args.context + W + K // 2)
                    r[f"decode_b{b}"] = {"tokens_per_s": round(d["tokens_per_s"], 1), "ms_per_step": round(d["ms_per_step"], 4),
                                         "hbm_frac": round(nbytes / (d["ms_per_step"] * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}
                kinds = (("parallel", 0), ("recurrent", 1)) if arm == "redudra" and layers > 1 else (("", 0),)
                for kind, layer in kinds:
                    for label, ql, kl in (("prefill_2048", [2048], [2048]), ("decode_b64", [1] * 64, [args.context] * 64)):
                        parts = B.time_parts(runner, ql, kl, layer=layer)
                        for part, v in parts.items():
                            sec = v["ms"] * 1e-3
                            r[f"{kind + '_' if kind else ''}{part}_{label}"] = {
                                "us": round(v["ms"] * 1e3, 1),
                                "tflops_frac": round(v["flops"] / sec / (pk["bf16_tflops"] * 1e12), 4),
                                "hbm_frac": round(v["bytes"] / sec / 1e9 / pk["hbm_gbs"], 4)}
            except B.Refused as exc:
                r["refused"] = str(exc)
            res[arm + "_result"] = r
            del runner, model
            _free_device_memory()
        out["sizes"][name] = res
    print(json.dumps(out))
    return 0


def run_design(args) -> int:
    """``--design zotonex``: prefill and decode throughput of the Zotonex design at layer sizes of real models (random
    weights, a few layers), beside a Qwen3 model of equal size: the same width, as many heads of the same value size,
    and an intermediate size equal to what a Zotonex token's experts add up to (top * ff + shared ff).  Whole steps
    through the step function, and one layer's mixer and feed-forward alone with their rooflines (L2 flushed before
    each timed run).  One JSON line."""
    import torch

    from acvram_b200 import bench as B
    from acvram_b200.config import Qwen3Config, ZotonexConfig
    from acvram_b200.engine.runner import ModelRunner
    from acvram_b200.models import build_random

    pk, pk_src = peaks()
    K, W = args.steps, args.warmup
    page = 64
    layers, vocab = args.layers or 4, 32768
    out = {"design": "zotonex", "beside": "qwen3", "layers": layers, "vocab": vocab, "dtype": "bf16", "page_size": page,
           "data": "synthetic token ids, random weights", "peaks": {**pk, "source": pk_src}, "sizes": {}}
    for name in args.sizes.split(","):
        z = ZOTONEX_SIZES[name]
        layer = {"type": "attention",
                 "mixer": {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["vdim"], "diff": 0.5,
                           "scale": z["dim"] ** -0.5, "mask": {"size": z["chunk"]}},
                 "mlp": {"kind": "moe", "router": {"experts": z["experts"], "top": z["top"]}, "expert": {"ff": z["ff"], "limit": 7.0},
                         "shared": {"ff": z["shared_ff"], "limit": 7.0}}}
        zcfg = ZotonexConfig.from_dict({"architecture": "Zotonex", "vocab": vocab, "width": z["width"], "norm": {"eps": 1e-5},
                                        "embedding": {"scale": 1.0}, "logit_scale": 1.0, "layers": [layer] * layers})
        qcfg = Qwen3Config(vocab_size=vocab, hidden_size=z["width"], intermediate_size=z["top"] * z["ff"] + z["shared_ff"],
                           num_hidden_layers=layers, num_attention_heads=z["heads"], num_key_value_heads=z["kv_heads"],
                           head_dim=z["vdim"], rms_norm_eps=1e-6, rope_theta=1e6, max_position_embeddings=8192,
                           tie_word_embeddings=False)
        res = {"zotonex": dict(z), "qwen3": {"hidden": qcfg.hidden_size, "intermediate": qcfg.intermediate_size,
                                            "q_heads": qcfg.num_attention_heads, "kv_heads": qcfg.num_key_value_heads,
                                            "head_dim": qcfg.head_dim}}
        for arm, cfg in (("zotonex", zcfg), ("qwen3", qcfg)):
            model = build_random(cfg, seed=0, dtype=torch.bfloat16, device="cuda:0")
            batch_max = 64
            tokens = batch_max * (args.context + 2 * (K + W) + 2 * page) + 4096
            runner = ModelRunner(model, page, tokens // page + 8, batch_max + 2, max_len=8192)
            if not args.no_cuda_graphs:
                runner.enable_graphs()
            r = {"weights_gb": round(model.weight_bytes() / 1e9, 3)}
            try:
                pre = B.time_prefill(runner, 2048, reps=5, warmup=3)
                flops = B.prefill_flops(model, 2048)
                r["prefill_2048"] = {"tokens_per_s": round(pre["tokens_per_s"], 1), "ms": round(pre["ms"], 3),
                                     "tflops_frac": round(flops / (pre["ms"] * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)}
                for b in (8, 64):
                    names = [f"d{b}-{i}" for i in range(b)]
                    B.fill_contexts(runner, names, args.context)
                    try:
                        d = B.time_decode(runner, names, K, W)
                    finally:
                        for n in names:
                            runner.release(n)
                    nbytes = B.decode_step_bytes(model, b, args.context + W + K // 2)
                    r[f"decode_b{b}"] = {"tokens_per_s": round(d["tokens_per_s"], 1), "ms_per_step": round(d["ms_per_step"], 4),
                                         "hbm_frac": round(nbytes / (d["ms_per_step"] * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}
                # one layer's parts alone: a prompt of 2048 tokens (bound by the tensor cores) and 64 requests that
                # decode at 2048-token contexts (bound by memory)
                for label, ql, kl in (("prefill_2048", [2048], [2048]), ("decode_b64", [1] * 64, [args.context] * 64)):
                    parts = B.time_parts(runner, ql, kl)
                    for part, v in parts.items():
                        sec = v["ms"] * 1e-3
                        r[f"{part}_{label}"] = {"us": round(v["ms"] * 1e3, 1),
                                                "tflops_frac": round(v["flops"] / sec / (pk["bf16_tflops"] * 1e12), 4),
                                                "hbm_frac": round(v["bytes"] / sec / 1e9 / pk["hbm_gbs"], 4)}
            except B.Refused as exc:
                r["refused"] = str(exc)
            res[arm + "_result"] = r
            del runner, model
            _free_device_memory()
        out["sizes"][name] = res
    print(json.dumps(out))
    return 0


def bench_config(args, cfg, layers: int, full_layers: int, page: int, graphs: bool) -> dict:
    """The configuration's sizes, flat, the same keys in both arms (the reference arm fills what it knows)."""
    return {"model": f"Qwen3-{args.shape.upper()} shape", "layers": layers, "layers_full": full_layers, "hidden": cfg["hidden_size"],
            "q_heads": cfg["num_attention_heads"], "kv_heads": cfg["num_key_value_heads"], "head_dim": cfg["head_dim"],
            "intermediate": cfg["intermediate_size"], "vocab": cfg["vocab_size"], "global_batch": args.batch,
            "seq_len": args.context, "max_model_len": 8192, "page_size": page, "kv_dtype": "bf16",
            "prefill_tokens": 2048, "parallelism": "single GPU",
            "l2": "inputs larger than L2 (weights + cache read per step >> 126 MB)", "cuda_graphs": graphs}


def main() -> int:
    ap = argparse.ArgumentParser(description=__doc__.split("\n\n")[0])
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=5)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--layers", type=int, default=0, help="fewer layers than the configuration's (named in config)")
    ap.add_argument("--shape", default="8b", choices=sorted(SHAPES), help="layer sizes (default: Qwen3-8B's)")
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--context", type=int, default=2048)
    ap.add_argument("--page-size", type=int, default=16, help="tokens in a page of the cache (the engine's own default is 64)")
    ap.add_argument("--skip-points", action="store_true", help="skip the batch 1 and 64 points")
    ap.add_argument("--no-cuda-graphs", action="store_true")
    ap.add_argument("--design", default="", choices=["", "zotonex", "redudra", "nizedra", "vadelix", "lodalix", "zogapel"],
                    help="measure another design beside its closest relative instead of the headline (see run_design)")
    ap.add_argument("--sizes", default="s,m", help="with --design: which of its sizes (s: width 2048, m: width 4096)")
    ap.add_argument("--time-limit", type=float, default=240.0,
                    help="seconds after which the points at the 14B and 32B layer sizes are left out (and named as left out)")
    args = ap.parse_args()
    if args.gpus != 1:
        print(f"bench.py measures one GPU; --gpus {args.gpus} is not built (the engine runs on a single device)")
        return 2
    if args.warmup < 3:
        args.warmup = 3
    if args.impl == "reference":
        return run_reference(args)
    if args.design == "redudra":
        return run_redudra(args)
    if args.design == "nizedra":
        return run_nizedra(args)
    if args.design == "vadelix":
        return run_vadelix(args)
    if args.design == "lodalix":
        return run_lodalix(args)
    if args.design == "zogapel":
        return run_zogapel(args)
    if args.design:
        return run_design(args)
    return run_ours(args)


if __name__ == "__main__":
    sys.exit(main())
