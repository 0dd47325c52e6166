"""Benchmark of the engine's decode step and prefill at Qwen3 layer sizes with random
weights, on one GPU.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference]
                    [--size 8b|14b|32b] [--workload decode|mixed] [--layers L]

A "step" is one decode step of a batch of 8 requests whose context is 2,048 prompt tokens
plus what they have generated. The region of K steps is timed with CUDA events and repeated;
`value` is decoded tokens a second at the median repeat. `e2e` is the same metric over K
steps by the wall clock through the Python entry point (`Engine.step`: host token ids in,
host token ids out, with the host-to-device copy of the step's batch from pinned memory and
the device-to-host read of the sampled tokens inside the timed region), also the median of
the repeats. Also on the line: one 2,048-token prefill with its share of the measured bf16
peak, the decode step's share of the measured HBM bandwidth with the bytes it counts, and
decode speed at batch 1 and 64. Weights (15 GB and more) are far larger than L2, so nothing
is flushed between steps. SM clocks and throttle reasons are sampled over all repeats.

`--size` selects the layer sizes (8b is the headline; 14b and 32b are the further sizes of
the benchmark configuration list). `--workload mixed` runs a continuous batch instead: 32
requests, prompt lengths uniform in [64, 3072], 128 to 512 new tokens each, Poisson arrivals,
half of them sharing a 1,024-token prefix, and reports generated tokens a second.

`--impl reference` runs the unmodified reference through its own Python primitive API and
Triton kernels (baseline/reference_arm.py) on the same metric and configuration.

`--design mugizen` measures another architecture of the engine instead of the headline: the
Mugizen design (parallel blocks of sink attention beside a gated delta rule over a float32
stream) at layer sizes that resemble a real model's (`--design-sizes s,m,moe`), beside Qwen3 at
the same width, heads, feed-forward width, layer count and vocabulary: one 2,048-token prefill
and decode steps at batch 8 and 1 for each, with their shares of the measured peaks.

`--design vivesun` does the same for the Vivesun design (pre-norm layers over a float32 stream,
gated-delta layers alternating with layers of chunked rotary attention beside a generalized
delta rule, an expert feed-forward in every layer) beside Mugizen, the engine's closest
model, at the same sizes.

`--design beralix` does the same for the Beralix design (layers normed before and after every
sublayer over a float32 stream: latent attention, windowed attention with value mixing and a
selective scan in turn, dense feed-forwards) beside Mugizen with dense feed-forwards at the
same sizes (`--design-sizes s,m`).
`--design nefipel` does the same for the Nefipel design (post-norm layers over a float32 stream,
gated attention and differential attention in turn, dense feed-forwards or, with size moe,
experts chosen by corrected scores with identity experts and a shared expert) beside Qwen3
(beside Mugizen where there are experts).

`--design pubulix` does the same for the Pubulix design (gated pre-norm layers over a float32 stream
with an input convolution: windowed latent attention, capped windowed attention, latent attention
over the first layer's latents, and capped attention again, clamped experts by token table in every
layer) beside Beralix, whose attention is closest (at sizes s and m, whose dense feed-forward does the
work of the two experts a token has), and beside Mugizen's experts (size moe).
`--design difavik` does the same for the Difavik design (output norms over a float32 stream, windowed attention
with linear penalties and kept first tokens beside retention, lightning attention, clamped feed-forwards with
biases or experts by a plain softmax) beside Mugizen at the same sizes (`--design-sizes s,m,moe`).
"""
from __future__ import annotations

import argparse
import json
import math
import os
import statistics
import subprocess
import sys
import tempfile
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)


def qwen3(layers, hidden, heads, kv_heads, inter, context=4096):
    return dict(
        architectures=["Qwen3ForCausalLM"], model_type="qwen3", num_hidden_layers=layers, hidden_size=hidden,
        num_attention_heads=heads, num_key_value_heads=kv_heads, head_dim=128, intermediate_size=inter,
        vocab_size=151936, rope_theta=1000000.0, rms_norm_eps=1e-6, tie_word_embeddings=False,
        max_position_embeddings=context, hidden_act="silu", attention_bias=False, attention_dropout=0.0,
        use_sliding_window=False, sliding_window=None, rope_scaling=None,
    )


SIZES = {
    "8b": ("Qwen3-8B size", qwen3(36, 4096, 32, 8, 12288)),
    "14b": ("Qwen3-14B size", qwen3(40, 5120, 40, 8, 17408)),
    "32b": ("Qwen3-32B size", qwen3(64, 5120, 64, 8, 25600)),
}
CONTEXT, PAGE = 2048, 16
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0}
MIN_TIMED_MS = 1200.0     # repeats of the K-step region go on until this much was timed (clock samples)


def load_peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.isfile(path):
        with open(path) as handle:
            return json.load(handle), "measured"
    return dict(FALLBACK_PEAKS), "fallback"


class ClockSampler:
    """nvidia-smi in the background while a region is timed."""

    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")
    NAMES = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]

    def __init__(self):
        self.file = tempfile.NamedTemporaryFile("w+", suffix=".csv", delete=False)
        self.proc = None

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", "0", f"--query-gpu={self.QUERY}",
                                          "--format=csv,noheader,nounits", "-lms", "50"],
                                         stdout=self.file, stderr=subprocess.DEVNULL)
        except OSError:
            self.proc = None

    def stop(self):
        if self.proc is not None:
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()
        self.file.flush()
        self.file.seek(0)
        sm, top, reasons = [], 0.0, set()
        for line in self.file.read().splitlines():
            fields = [f.strip() for f in line.split(",")]
            if len(fields) != 6:
                continue
            try:
                sm.append(float(fields[0]))
                top = max(top, float(fields[1]))
            except ValueError:
                continue
            for name, value in zip(self.NAMES, fields[2:]):
                if value.lower().startswith("active"):
                    reasons.add(name)
        self.file.close()
        os.unlink(self.file.name)
        return {"sm_mhz": statistics.median(sm) if sm else None, "sm_max_mhz": top or None,
                "reasons": sorted(reasons), "samples": len(sm)}


def random_prompts(count, length, vocab, seed):
    import torch
    gen = torch.Generator().manual_seed(seed)
    return [torch.randint(0, vocab, (length,), generator=gen).tolist() for _ in range(count)]


def repeats_for(steps, ms_per_step, least, most):
    return max(1, min(most, max(least, math.ceil(MIN_TIMED_MS / max(steps * ms_per_step, 1e-3)))))


DECODE_STEPS = 256        # a request decodes this many tokens in the benchmark's workload


def decode_run(engine, batch, steps, warmup, seed, sample_clocks=False, least_repeats=5):
    """Prefill `batch` requests of CONTEXT tokens, then time regions of `steps` decode steps:
    with CUDA events (device) and by the wall clock through Engine.step (end to end). Each
    region is repeated (at most DECODE_STEPS steps in all, so the context stays near CONTEXT)
    and the median is reported."""
    import torch
    from vosti_b200 import ops

    vocab = engine.runner.spec.vocab_size
    first = len(engine.scheduler.accepted_ids)
    budget = engine.runner.spec.max_positions - CONTEXT
    for i, prompt in enumerate(random_prompts(batch, CONTEXT, vocab, seed)):
        status = engine.add_request(first + i, prompt, budget, None, True)
        assert status.value == "accepted", status
    while any(not r.is_decoding() for r in engine.scheduler.running) or engine.scheduler.waiting:
        engine.step()
    assert len(engine.scheduler.running) == batch
    engine.step()                          # with async scheduling the first decode step's tokens come a call later
    for _ in range(warmup):
        assert len(engine.step()) == batch
    sampler = ClockSampler() if sample_clocks else None
    if sampler:
        sampler.start()
    context_start = engine.scheduler.running[0].computed
    begin, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    device_ms, launches, repeats = [], 0, max(1, min(least_repeats, DECODE_STEPS // steps))
    while len(device_ms) < repeats:
        launches_before = ops.LAUNCHES
        torch.cuda.synchronize()
        begin.record()
        for _ in range(steps):
            emitted = engine.step()
        end.record()
        torch.cuda.synchronize()
        device_ms.append(begin.elapsed_time(end) / steps)
        launches = ops.LAUNCHES - launches_before
        assert len(emitted) == batch
        if len(device_ms) == 1:
            repeats = repeats_for(steps, device_ms[0], least_repeats, max(1, DECODE_STEPS // steps))
    # the end-to-end regions stay inside the same key-length bucket of the decode graphs
    room = (CONTEXT // 512 + 1) * 512 - (context_start + repeats * steps) - 8
    wall_ms = []
    for _ in range(max(1, min(repeats, room // steps))):
        torch.cuda.synchronize()
        wall = time.perf_counter()
        for _ in range(steps):
            emitted = engine.step()
        torch.cuda.synchronize()
        wall_ms.append((time.perf_counter() - wall) * 1e3 / steps)
    clocks = sampler.stop() if sampler else None
    h2d = engine.runner.staging.last_upload_bytes
    d2h = 4 * (1 + batch)
    context_mid = context_start + repeats * steps // 2
    for i in range(batch):
        engine.abort(first + i)
    engine.drain()
    assert not engine.has_unfinished()
    return {"device_ms": statistics.median(device_ms), "wall_ms": statistics.median(wall_ms), "launches": launches,
            "clocks": clocks, "h2d": h2d, "d2h": d2h, "context": context_mid, "repeats": repeats}


def prefill_run(engine, repeats, seed):
    """One CONTEXT-token prompt in one step, timed with CUDA events; the median of `repeats`
    runs after one that is not counted."""
    import torch

    vocab = engine.runner.spec.vocab_size
    times = []
    for r, prompt in enumerate(random_prompts(repeats + 1, CONTEXT, vocab, seed)):
        rid = len(engine.scheduler.accepted_ids)
        engine.add_request(rid, prompt, 1, None, True)
        begin, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        begin.record()
        emitted = engine.step()
        end.record()
        torch.cuda.synchronize()
        emitted.update(engine.drain())
        assert rid in emitted and not engine.has_unfinished()
        times.append(begin.elapsed_time(end))
    return statistics.median(times[1:])


def flops_of_prefill(config, tokens):
    L, H = config["num_hidden_layers"], config["hidden_size"]
    nq, nkv, d, I, V = (config["num_attention_heads"], config["num_key_value_heads"], config["head_dim"],
                        config["intermediate_size"], config["vocab_size"])
    linear = 2.0 * tokens * L * (H * (nq + 2 * nkv) * d + nq * d * H + 3 * H * I) + 2.0 * V * H
    attention = L * nq * d * 4.0 * tokens * (tokens + 1) / 2
    return linear + attention


def closed_form_weight_bytes(config):
    """bf16 bytes of every weight a decode step reads whole: per layer the four attention
    projections, two head norms, two norms, three feed-forward matrices; the final norm; the
    output head (the embedding table is read by rows, one per token)."""
    L, H = config["num_hidden_layers"], config["hidden_size"]
    nq, nkv, d, I, V = (config["num_attention_heads"], config["num_key_value_heads"], config["head_dim"],
                        config["intermediate_size"], config["vocab_size"])
    per_layer = H * (nq + 2 * nkv) * d + nq * d * H + 3 * H * I + 2 * H + 2 * d
    return 2 * (L * per_layer + H + V * H)


def reference_main(args) -> int:
    """The reference arm: same metric, same configuration, the reference's own code."""
    name, config = SIZES[args.size]
    try:
        if args.size != "8b":
            raise RuntimeError(f"the reference has launch profiles for qwen3-0.6b and qwen3-8b only, not {args.size}")
        import torch
        from baseline import reference_arm as arm
        peaks, peak_kind = load_peaks()
        layers = args.layers or config["num_hidden_layers"]
        max_batch = args.batch if args.no_points else max(args.batch, 64)
        per_request = CONTEXT + 64 * 3
        model = arm.ReferenceModel("qwen3-8b", layers, max_batch * per_request + 128, seed=0)
        ref_config = dict(model.config)
        ref_config["num_hidden_layers"] = layers
        prefill_ms = float("nan") if args.no_prefill else arm.prefill_run(model, CONTEXT, 3, seed=11)
        sampler = ClockSampler()
        sampler.start()
        runs = [arm.decode_run(model, args.batch, CONTEXT, args.steps, args.warmup, seed=21)
                for _ in range(1 if args.steps * 2 + args.warmup + 2 > 60 else 3)]
        clocks = sampler.stop()
        main_run = sorted(runs, key=lambda r: r["device_ms"])[len(runs) // 2]
        points = {}
        if not args.no_points:
            for batch in (1, 64):
                run = arm.decode_run(model, batch, CONTEXT, max(8, min(args.steps // 2, 24)), 3, seed=31 + batch)
                points[f"decode_b{batch}"] = round(batch * 1e3 / run["device_ms"], 1)
        step_bytes = model.weight_bytes + args.batch * main_run["context"] * model.kv_bytes_per_token
        achieved = step_bytes / (main_run["device_ms"] * 1e-3) / 1e9
        tflops = flops_of_prefill(ref_config, CONTEXT) / (prefill_ms * 1e-3) / 1e12
        line = {
            "metric": f"decode tok/s at batch {args.batch} ({name}, context {CONTEXT})",
            "value": round(args.batch * 1e3 / main_run["device_ms"], 1), "unit": "tok/s", "n_gpus": 1,
            "steps": args.steps, "warmup": args.warmup, "ms_per_step": round(main_run["device_ms"], 4),
            "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16",
            "data": "synthetic: random token ids, random-init weights", "impl": "reference",
            "config": {"model": name, "layers": layers, "layers_full": config["num_hidden_layers"],
                       "hidden": ref_config["hidden_size"], "heads": ref_config["num_attention_heads"],
                       "kv_heads": ref_config["num_key_value_heads"], "head_dim": ref_config["head_dim"],
                       "intermediate": ref_config["intermediate_size"], "vocab": ref_config["vocab_size"],
                       "global_batch": args.batch, "seq_len": CONTEXT, "page_size": arm.PAGE, "parallelism": "1 GPU",
                       "path": "vosti_kernels primitives + Triton kernels + CudaGraphOverlay, Python host loop",
                       "l2": "inputs larger than L2 (weights read every step)", "peaks": peak_kind},
            "e2e": {"value": round(args.batch * 1e3 / main_run["wall_ms"], 1), "unit": "tok/s",
                    "h2d_bytes_per_step": main_run["h2d"], "d2h_bytes_per_step": main_run["d2h"]},
            "clocks": clocks,
            "prefill": {"value": round(CONTEXT * 1e3 / prefill_ms, 1), "tokens": CONTEXT, "ms": round(prefill_ms, 3),
                        "frac": round(tflops / peaks["bf16_tflops"], 4),
                        "frac_of_sustained": round(tflops / peaks.get("bf16_tflops_sustained", peaks["bf16_tflops"]), 4)},
            "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": peaks["hbm_gbs"], "unit": "GB/s",
                         "frac": round(achieved / peaks["hbm_gbs"], 4), "bytes_per_step": int(step_bytes)},
            "points": points,
        }
        print(json.dumps(line))
    except Exception as error:  # the arm must report, not crash: the driver reads this line
        import traceback
        traceback.print_exc(file=sys.stderr)
        text = " ".join(f"{type(error).__name__}: {error}".split())
        print(json.dumps({"impl": "reference", "unavailable": text[:600]}))
    return 0


def mixed_run(engine, config, seed=5, requests=32, rate_per_s=16.0):
    """A continuous batch: `requests` prompts with lengths uniform in [64, 3072] and 128 to 512
    new tokens each, Poisson arrivals at `rate_per_s`, half of them starting with the same
    1,024 tokens. Returns generated tokens, wall seconds and what the cache reused."""
    import random
    import torch

    rng = random.Random(seed)
    vocab = config["vocab_size"]
    gen = torch.Generator().manual_seed(seed)
    draw = lambda n: torch.randint(0, vocab, (n,), generator=gen).tolist()
    shared = draw(1024)
    plan, at = [], 0.0
    for i in range(requests):
        length = rng.randint(64, 3072)
        new_tokens = rng.randint(128, 512)
        prompt = (shared + draw(max(length - 1024, 1))) if i % 2 == 0 else draw(length)
        at += rng.expovariate(rate_per_s)
        plan.append((at, i, prompt, new_tokens))
    first = len(engine.scheduler.accepted_ids)
    generated, first_token_at, arrived_at = 0, {}, {}
    torch.cuda.synchronize()
    start = time.perf_counter()
    steps = 0
    while plan or engine.has_unfinished():
        now = time.perf_counter() - start
        while plan and plan[0][0] <= now:
            _, i, prompt, new_tokens = plan.pop(0)
            status = engine.add_request(first + i, prompt, new_tokens, None, True)
            assert status.value == "accepted", status
            arrived_at[first + i] = now
        if not engine.has_unfinished():
            time.sleep(max(0.0, plan[0][0] - now))
            continue
        emitted = engine.step()
        steps += 1
        generated += len(emitted)
        now = time.perf_counter() - start
        for rid in emitted:
            first_token_at.setdefault(rid, now)
    torch.cuda.synchronize()
    wall = time.perf_counter() - start
    ttft = sorted(first_token_at[r] - arrived_at[r] for r in first_token_at)
    return {"generated": generated, "wall_s": wall, "steps": steps, "ttft_median_s": ttft[len(ttft) // 2],
            "ttft_max_s": ttft[-1], **engine.cache_stats()}


# ---------------------------------------------------------------- another design beside Qwen3
DESIGN_SIZES = {
    # width, heads, kv heads (head size 128 everywhere), feed-forward, layers, vocabulary, experts
    "s": dict(width=2048, heads=16, kv=4, ff=8192, layers=4, vocab=32768, moe=None),
    "m": dict(width=4096, heads=32, kv=8, ff=12288, layers=4, vocab=32768, moe=None),
    "moe": dict(width=2048, heads=16, kv=4, ff=8192, layers=4, vocab=32768, moe=dict(experts=8, top=2, ff=4096)),
}


def mugizen_config(size):
    """A Mugizen config.json of these sizes (no layer loop, so that a layer runs once as Qwen3's do)
    and the tensor shapes that give the sizes the config leaves out."""
    from vosti_b200.config.mugizen import checkpoint_shapes
    left = dict(heads=size["heads"], kv_heads=size["kv"], dim=128, vdim=128, scale=128 ** -0.5, bias_max=1024,
                q_temp=dict(coef=0.1, every=1024))
    right = dict(heads=size["heads"], kv_heads=size["kv"], dim=128, vdim=128, conv=4)
    if size["moe"]:
        mlp = dict(kind="moe", expert=dict(ff=size["moe"]["ff"]), router=dict(experts=size["moe"]["experts"], top=size["moe"]["top"]))
    else:
        mlp = dict(kind="dense", ff=size["ff"])
    config = dict(architecture="Mugizen", vocab=size["vocab"], width=size["width"], norm=dict(eps=1e-6), loop=None,
                  layers=[dict(type="parallel", mixer=dict(left=left, right=right), mlp=mlp) for _ in range(size["layers"])])
    return config, checkpoint_shapes(config, bias_rows=32, decay_rank=64, gate_rank=64)


def vivesun_config(size):
    """A Vivesun config.json of these sizes: gated-delta layers and parallel layers in turn, every
    layer with an expert feed-forward (two of eight experts; where the size names a dense
    feed-forward the experts are 3/4 of its width, so that a token's two two-matrix experts do
    the work of one three-matrix feed-forward), and the shape that gives the decay pair's rank."""
    from vosti_b200.config.vivesun import checkpoint_shapes
    moe = size["moe"] or dict(experts=8, top=2, ff=size["ff"] * 3 // 4)
    mlp = dict(kind="moe", expert=dict(ff=moe["ff"]), router=dict(experts=moe["experts"], top=moe["top"], scale=1.0))
    left = dict(heads=size["heads"], kv_heads=size["kv"], dim=128, vdim=128, scale=128 ** -0.5, mask=dict(size=1024),
                rot=dict(base=500000.0, dims=64, scaling=dict(factor=8.0, low=1.0, high=4.0, original=8192)))
    parallel = dict(type="parallel", mlp=mlp, mixer=dict(left=left, right=dict(heads=size["heads"], dim=128),
                                                         left_scale=1.0, right_scale=1.0))
    delta = dict(type="delta", mlp=mlp, mixer=dict(heads=size["heads"], kv_heads=size["kv"], dim=128, vdim=128, conv=4))
    config = dict(architecture="Vivesun", vocab=size["vocab"], width=size["width"], norm=dict(eps=1e-6), token_side=dict(dim=64),
                  embedding=dict(bigram=dict(buckets=65521, mul_prev=1000003, mul_cur=31)),
                  layers=[delta if i % 2 == 0 else parallel for i in range(size["layers"])])
    return config, checkpoint_shapes(config, decay_rank=64)


def vivesun_flops(size, tokens):
    """Multiply-add work of one prompt, times two, for `vivesun_config(size)`."""
    W, H, G, L, V, d = size["width"], size["heads"], size["kv"], size["layers"], size["vocab"], 128
    moe = size["moe"] or dict(experts=8, top=2, ff=size["ff"] * 3 // 4)
    feed = 2 * W * moe["ff"] * moe["top"] + W * moe["experts"] + 2 * W * 64            # experts, router, token input
    delta = W * (2 * G * d + H * d + H) + W * (H + H * d) + H * d * W                  # q | k | v | beta, a | g, o
    parallel = W * (H + 2 * G) * d + H * d * W + W * (5 * H * d + 64) + 64 * H * d + H * d * W
    per_token = (L - L // 2) * (delta + feed) + (L // 2) * (parallel + feed)
    chunk = min(tokens, 1024)
    scores = (L // 2) * H * d * 4.0 * tokens * (chunk + 1) / 2                          # a query sees at most its chunk
    state = L * tokens * H * 4.0 * d * d                                               # 4 passes over a 128 x 128 state
    return 2.0 * tokens * per_token + 2.0 * V * W + scores + state


def beralix_config(size):
    """A Beralix config.json of these sizes: latent attention (a latent of 512, 64 rotated and 128
    unrotated elements a head), windowed attention (window 1,024, whole-head rescaled rotation),
    a selective scan (twice the width, 16 states, 4 taps) and windowed attention again; the two
    windowed layers mix values. Every layer has a dense feed-forward."""
    H, G, W = size["heads"], size["kv"], size["width"]
    yarn = dict(factor=8.0, original=4096, fast=32.0, slow=1.0)
    mlp = dict(kind="dense", ff=size["ff"])
    latent = dict(type="latent_attention", mlp=mlp, mixer=dict(heads=H, dim=128, rot_dim=64, vdim=128, kv_rank=512, scale=192 ** -0.5,
                                                               rot=dict(base=10000.0, dims=64, scaling=yarn)))
    window = dict(type="attention", mlp=mlp, mixer=dict(heads=H, kv_heads=G, dim=128, vdim=128, scale=128 ** -0.5, mask=dict(size=1024),
                                                        v_mix=True, rot=dict(base=500000.0, dims=128, scaling=yarn)))
    scan = dict(type="mamba1", mlp=mlp, mixer=dict(inner=2 * W, state=16, conv=4, dt_rank=W // 16))
    order = [latent, window, scan, window]
    return dict(architecture="Beralix", vocab=size["vocab"], width=W, norm=dict(eps=1e-5), logit_softcap=30.0,
                layers=[order[i % 4] for i in range(size["layers"])])


def beralix_flops(size, tokens):
    """Multiply-add work of one prompt, times two, for `beralix_config(size)`, as the engine computes
    it: the latent attention scores and sums over the cached latents (rank + rotated elements a key
    for the score, rank for the sum), after carrying the query into the latent space."""
    W, H, G, F, L, V, d = size["width"], size["heads"], size["kv"], size["ff"], size["layers"], size["vocab"], 128
    rank, rot, inner, N, low = 512, 64, 2 * W, 16, W // 16
    latent = W * (H * (d + rot) + rank + rot + H) + 2 * H * d * rank + H * d * W
    window = W * (H + 2 * G) * d + H * d * W
    scan = W * 2 * inner + inner * (low + 2 * N) + low * inner + inner * W + 3 * inner * N
    kinds = [latent, window, scan, window]
    per_token = sum(kinds[i % 4] + 3 * W * F for i in range(L))
    pairs_all = tokens * (tokens + 1) / 2
    pairs_window = sum(min(t + 1, 1024) for t in range(tokens))
    scores = sum((H * (2 * rank + rot) * 2.0 * pairs_all) if i % 4 == 0 else (H * d * 4.0 * pairs_window) if i % 4 in (1, 3) else 0.0
                 for i in range(L))
    return 2.0 * tokens * per_token + 2.0 * V * W + scores


def nefipel_config(size):
    """A Nefipel config.json of these sizes: gated attention (heads of 128, half of each head rotated)
    and differential attention (two maps of 64 a head over values of 128, whole-map rescaled
    rotation) in turn. Feed-forwards are dense, or with size "moe" the differential layers have the
    size's experts (two of them chosen, among the experts and two identity experts in two groups of
    which one is kept) and a shared expert as wide as one expert."""
    H, G, W = size["heads"], size["kv"], size["width"]
    yarn = dict(factor=8.0, original=4096, fast=32.0, slow=1.0)
    dense = dict(kind="dense", ff=size["ff"])
    sparse = dense
    if size["moe"]:
        m = size["moe"]
        sparse = dict(kind="moe", expert=dict(ff=m["ff"]), shared=dict(ff=m["ff"]),
                      router=dict(experts=m["experts"], top=m["top"], identity=2, groups=dict(count=2, keep=1)))
    gated = dict(type="attention", mlp=dense, mixer=dict(heads=H, kv_heads=G, dim=128, vdim=128, scale=128 ** -0.5,
                                                         rot=dict(base=10000.0, dims=64)))
    diff = dict(type="attention_2", mlp=sparse, mixer=dict(heads=H, kv_heads=G, dim=64, vdim=128, scale=64 ** -0.5, diff=0.3,
                                                           rot=dict(base=500000.0, dims=64, scaling=yarn)))
    return dict(architecture="Nefipel", vocab=size["vocab"], width=W, norm=dict(eps=1e-5), postln_alpha=2.0,
                embedding=dict(scale=W ** 0.5), layers=[(gated, diff)[i % 2] for i in range(size["layers"])])


def nefipel_flops(size, tokens):
    """Multiply-add work of one prompt, times two, for `nefipel_config(size)`: products (of the experts,
    those a token chooses and the shared one) and both maps' scores and weighted sums."""
    W, H, G, F, L, V = size["width"], size["heads"], size["kv"], size["ff"], size["layers"], size["vocab"]
    gated = W * (H + 2 * G) * 128 + W * H * 128 + H * 128 * W             # q | k | v, the gate, the output
    diff = W * (2 * H * 64 + 2 * G * 64 + G * 128) + H * 128 * W
    sparse = 3 * W * F
    if size["moe"]:
        m = size["moe"]
        sparse = 2 * W * m["ff"] * (m["top"] + 1) + W * (m["experts"] + 3)
    per_token = sum((gated + 3 * W * F) if i % 2 == 0 else (diff + sparse) for i in range(L))
    pairs = tokens * (tokens + 1) / 2
    scores = sum(H * (128 * 4.0 if i % 2 == 0 else (2 * 64 + 2 * 128) * 2.0) * pairs for i in range(L))
    return 2.0 * tokens * per_token + 2.0 * V * W + scores


def pubulix_experts(size):
    """The size's experts, or eight of half the dense feed-forward's width of which a token has two."""
    return size["moe"] or dict(experts=8, top=2, ff=size["ff"] // 2)


def pubulix_config(size):
    """A Pubulix config.json of these sizes: latent attention (a latent of 512, 64 rotated and 128
    unrotated elements a head) that keeps its own latents, capped grouped-query attention, latent
    attention over the first layer's latents, capped attention; windows of 1,024; four taps."""
    H, G, W, m = size["heads"], size["kv"], size["width"], pubulix_experts(size)
    mlp = dict(kind="moe", expert=dict(ff=m["ff"], limit=7.0), router=dict(experts=m["experts"], top=m["top"]))
    latent = dict(heads=H, dim=128, rot_dim=64, vdim=128, kv_rank=512, scale=192 ** -0.5, mask=dict(size=1024),
                  rot=dict(base=10000.0, dims=64))
    capped = dict(type="attention", mlp=mlp, mixer=dict(heads=H, kv_heads=G, dim=128, vdim=128, scale=128 ** -0.5, softcap=50.0,
                                                        mask=dict(size=1024), rot=dict(base=10000.0, dims=128)))
    order = [dict(type="latent_attention", mlp=mlp, mixer=latent), capped,
             dict(type="latent_attention", mlp=mlp, mixer=dict(latent, kv_from=0)), capped]
    return dict(architecture="Pubulix", vocab=size["vocab"], width=W, norm=dict(eps=1e-5), canon=dict(taps=4), residual_mult=0.5,
                embedding=dict(scale=W ** 0.5), logit_softcap=30.0, layers=[order[i % 4] for i in range(size["layers"])])


def pubulix_flops(size, tokens):
    """Multiply-add work of one prompt, times two, for `pubulix_config(size)`, the latent attention as the
    engine computes it (scores and sums over the cached latents)."""
    W, H, G, L, V, d = size["width"], size["heads"], size["kv"], size["layers"], size["vocab"], 128
    m, rank, rot, taps = pubulix_experts(size), 512, 64, 4
    query = W * H * (d + rot) + W * H * d + 2 * H * d * rank + H * d * W              # q, gate, into and out of the latent space, o
    kinds = [query + W * (rank + rot), W * (H + 2 * G) * d + H * d * W, query, W * (H + 2 * G) * d + H * d * W]
    per_token = sum(kinds[i % 4] + 2 * W * W + taps * W + 3 * W * m["ff"] * m["top"] for i in range(L))
    pairs = sum(min(t + 1, 1024) for t in range(tokens))
    scores = sum((H * (2 * rank + rot) * 2.0 if i % 2 == 0 else H * d * 4.0) * pairs for i in range(L))
    return 2.0 * tokens * per_token + 2.0 * V * W + scores


def difavik_config(size):
    """A Difavik config.json of these sizes: parallel layers (windowed attention whose values are its keys, a window
    of 1,024 and 64 kept tokens, beside retention) and lightning layers in turn, heads of 128 everywhere."""
    H, G, W = size["heads"], size["kv"], size["width"]
    if size["moe"]:
        mlp = dict(kind="moe", expert=dict(ff=size["moe"]["ff"], limit=7.0), router=dict(experts=size["moe"]["experts"], top=size["moe"]["top"]))
    else:
        mlp = dict(kind="dense", ff=size["ff"], limit=7.0)
    decay = [1.0 - 2.0 ** (-5.0 - 6.0 * h / H) for h in range(H)]
    parallel = dict(type="parallel", mlp=mlp, mixer=dict(
        left=dict(heads=H, kv_heads=G, dim=128, vdim=128, scale=128 ** -0.5, mask=dict(size=1024, keep_first=64)),
        right=dict(heads=H, dim=128, vdim=128, rot=dict(base=10000.0, dims=128), decay=decay)))
    light = dict(type="lightning", mlp=mlp, mixer=dict(heads=H, dim=128, vdim=128, decay=decay))
    return dict(architecture="Difavik", vocab=size["vocab"], width=W, norm=dict(eps=1e-5),
                embedding=dict(bigram=dict(buckets=65521, mul_prev=1000003, mul_cur=31)),
                layers=[parallel if i % 2 == 0 else light for i in range(size["layers"])])


def difavik_flops(size, tokens):
    """Multiply-add work of one prompt, times two, for `difavik_config(size)`."""
    W, H, G, L, V, d = size["width"], size["heads"], size["kv"], size["layers"], size["vocab"], 128
    feed = 3 * W * size["ff"] if not size["moe"] else 3 * W * size["moe"]["ff"] * size["moe"]["top"] + W * size["moe"]["experts"]
    recurrent, attention = 5 * W * H * d, W * ((H + G) * d + H) + H * d * W
    per_token = L * (recurrent + feed) + (L - L // 2) * attention
    pairs = sum(min(t + 1, 1024 + min(max(t - 1023, 0), 64)) for t in range(tokens))
    scores = (L - L // 2) * H * d * 4.0 * pairs + L * tokens * H * 4.0 * d * d       # attention; 2 passes over a 128 x 128 state
    return 2.0 * tokens * per_token + 2.0 * V * W + scores


def unread_bytes(size, batch):
    """Weight bytes of experts that a Pubulix or Difavik decode step of `batch` requests of random tokens does not read."""
    m = pubulix_experts(size)
    idle = (1.0 - m["top"] / m["experts"]) ** batch * m["experts"]
    return size["layers"] * idle * 3 * size["width"] * m["ff"] * 2.0


def design_flops(size, tokens, design):
    """Multiply-add work of one prompt of `tokens` tokens, times two: the products and the attention."""
    if design == "vivesun":
        return vivesun_flops(size, tokens)
    if design == "beralix":
        return beralix_flops(size, tokens)
    if design == "nefipel":
        return nefipel_flops(size, tokens)
    if design == "difavik":
        return difavik_flops(size, tokens)
    if design == "pubulix":
        return pubulix_flops(size, tokens)
    W, H, G, F, L, V = size["width"], size["heads"], size["kv"], size["ff"], size["layers"], size["vocab"]
    d = 128
    attention = W * (H + 2 * G) * d + H * d * W
    feed = 3 * W * F if not size["moe"] else 3 * W * size["moe"]["ff"] * size["moe"]["top"]
    per_token = attention + feed
    scores = L * H * d * 4.0 * tokens * (tokens + 1) / 2
    if design == "mugizen":
        # the recurrent branch: q | k | v | beta, the low-rank pairs (rank 64), the output projection,
        # and per token and head 4 passes over a 128 x 128 state
        per_token += W * (2 * G * d + H * d + H) + W * 128 + 128 * 2 * H * d + H * d * W
        scores += L * tokens * H * 4.0 * d * d
    return 2.0 * tokens * (L * per_token) + 2.0 * V * W + scores


def design_engine(kind, size, max_batch):
    import torch
    from vosti_b200 import Engine
    from vosti_b200.config import model_spec_from_config
    from vosti_b200.models import expected_weights
    from vosti_b200.weights import draw_tensors

    if kind == "mugizen":
        config, shapes = mugizen_config(size)
        spec = model_spec_from_config(config, shapes)
    elif kind == "vivesun":
        config, shapes = vivesun_config(size)
        spec = model_spec_from_config(config, shapes)
    elif kind == "beralix":
        spec = model_spec_from_config(beralix_config(size))
    elif kind == "nefipel":
        spec = model_spec_from_config(nefipel_config(size))
    elif kind == "difavik":
        spec = model_spec_from_config(difavik_config(size))
    elif kind == "pubulix":
        spec = model_spec_from_config(pubulix_config(size))
    else:
        spec = model_spec_from_config(qwen3(size["layers"], size["width"], size["heads"], size["kv"], size["ff"],
                                            context=CONTEXT + 2048) | {"vocab_size": size["vocab"]})
    tensors = draw_tensors(expected_weights(spec), seed=0, device=torch.device("cuda:0"), dtype=torch.bfloat16)
    tokens_per_request = CONTEXT + 2 * DECODE_STEPS + 128
    engine = Engine(spec=spec, tensors=tensors, dtype="bfloat16", device="cuda:0",
                    num_blocks=max_batch * ((tokens_per_request + PAGE - 1) // PAGE) + 8, block_size=PAGE,
                    max_num_seqs=max_batch, max_num_batched_tokens=2 * CONTEXT, enable_prefix_caching=False,
                    cuda_graphs=True, async_scheduling=True, consume_tensors=True)
    del tensors
    torch.cuda.empty_cache()
    return engine


def design_one(args, name, kind) -> dict:
    """One model (a size and a design) in this process: prefill, decode at batch 8 and 1."""
    import torch

    peaks, _ = load_peaks()
    torch.cuda.set_device(0)
    size = DESIGN_SIZES[name]
    print(f"[bench] {name}: {kind}: building", file=sys.stderr, flush=True)
    engine = design_engine(kind, size, 8)
    runner = engine.runner
    weight_bytes = runner.model.weight_bytes()
    kv_bytes = runner.cache.bytes_per_token()
    state_bytes = sum(c.state[0].numel() * c.state.element_size() for c in runner.cache.layer_caches if c.state is not None)
    print(f"[bench] {name}: {kind}: prefill", file=sys.stderr, flush=True)
    prefill_ms = prefill_run(engine, 3, seed=11)
    tflops = design_flops(size, CONTEXT, kind) / (prefill_ms * 1e-3) / 1e12
    entry = {"prefill_tok_s": round(CONTEXT * 1e3 / prefill_ms, 1), "prefill_ms": round(prefill_ms, 3),
             "prefill_frac_of_bf16_peak": round(tflops / peaks["bf16_tflops"], 4),
             "weight_bytes": int(weight_bytes), "kv_bytes_per_token": int(kv_bytes), "state_bytes": int(state_bytes)}
    for batch in (8, 1):
        print(f"[bench] {name}: {kind}: decode at batch {batch}", file=sys.stderr, flush=True)
        run = decode_run(engine, batch, args.steps, args.warmup, seed=21 + batch, least_repeats=3)
        kv_read = run["context"] * kv_bytes
        if kind == "pubulix":                   # windows of 1,024; the first layer's latents are read by two layers
            kv_read = min(run["context"], 1024) * (kv_bytes + 576 * 2 * ((size["layers"] + 1) // 4))
        if kind == "difavik":                   # a window of 1,024 and 64 kept tokens
            kv_read = min(run["context"], 1024 + 64) * kv_bytes
        step_bytes = weight_bytes + batch * (kv_read + 2 * state_bytes) - (unread_bytes(size, batch) if kind == "pubulix" else
                                                                                        unread_bytes(size, batch) if kind == "difavik" and size["moe"] else 0)
        entry[f"decode_b{batch}"] = {
            "tok_s": round(batch * 1e3 / run["device_ms"], 1), "ms_per_step": round(run["device_ms"], 4),
            "e2e_tok_s": round(batch * 1e3 / run["wall_ms"], 1), "launches_per_step": run["launches"] / args.steps,
            "frac_of_hbm_peak": round(step_bytes / (run["device_ms"] * 1e-3) / 1e9 / peaks["hbm_gbs"], 4)}
    return entry


BESIDE = {"mugizen": "qwen3", "vivesun": "mugizen", "beralix": "mugizen", "nefipel": "qwen3", "pubulix": "beralix", "difavik": "mugizen"}      # the engine's closest other model


def design_main(args) -> int:
    """Prefill and decode of a design beside the engine's closest other model (Mugizen beside Qwen3,
    Vivesun, Beralix and Difavik beside Mugizen, Pubulix beside Beralix) at equal sizes; one JSON line. Every
    model is measured in a process of its own (this program started again with --design-one), so
    that no model's scratch buffers, graphs or allocator state reach the next one's timings."""
    if args.design_one:
        name, kind = args.design_one.split(":")
        print(json.dumps(design_one(args, name, kind)))
        return 0
    _, peak_kind = load_peaks()
    out = {}
    for name in args.design_sizes.split(","):
        size = DESIGN_SIZES[name]
        if args.design == "beralix" and size["moe"]:
            continue                          # the design's feed-forwards are dense
        row = {}
        for kind in (args.design, BESIDE[args.design]):
            if kind == "qwen3" and size["moe"]:
                if args.design != "nefipel":
                    continue                  # the engine has no other model with experts to stand beside
                kind = "mugizen"              # Nefipel's experts stand beside Mugizen's
            if kind == "beralix" and args.design == "pubulix" and size["moe"]:
                kind = "mugizen"              # and so do Pubulix's
            child = subprocess.run([sys.executable, os.path.abspath(__file__), "--design", args.design, "--design-one",
                                    f"{name}:{kind}", "--steps", str(args.steps), "--warmup", str(args.warmup),
                                    "--context", str(CONTEXT), "--page", str(PAGE)],
                                   stdout=subprocess.PIPE, text=True, timeout=900)
            lines = [line for line in child.stdout.splitlines() if line.startswith("{")]
            if child.returncode != 0 or not lines:
                raise RuntimeError(f"measuring {kind} at size {name} failed (exit code {child.returncode})")
            row[kind] = json.loads(lines[-1])
        out[name] = {"sizes": {k: v for k, v in size.items()}, **row}
    print(json.dumps({"design": args.design, "beside": BESIDE[args.design] + " at equal sizes", "context": CONTEXT, "page_size": PAGE,
                      "steps": args.steps, "warmup": args.warmup, "dtype": "bf16", "peaks": peak_kind,
                      "data": "synthetic: random token ids, random-init weights", "results": out}))
    return 0


def main() -> int:
    parser = argparse.ArgumentParser()
    parser.add_argument("--gpus", type=int, default=1)
    parser.add_argument("--steps", type=int, default=64)
    parser.add_argument("--warmup", type=int, default=4)
    parser.add_argument("--impl", default="ours", choices=["ours", "reference"])
    parser.add_argument("--size", default="8b", choices=sorted(SIZES), help="layer sizes (8b is the headline)")
    parser.add_argument("--workload", default="decode", choices=["decode", "mixed"],
                        help="decode: the headline; mixed: a continuous batch with Poisson arrivals and a shared prefix")
    parser.add_argument("--layers", type=int, default=0, help="fewer layers than the configuration (both are reported)")
    parser.add_argument("--context", type=int, default=2048,
                        help="prompt length of the decode requests and of the prefill (the headline is 2048)")
    parser.add_argument("--page", type=int, default=16, help="tokens per cache page")
    parser.add_argument("--batch", type=int, default=8)
    parser.add_argument("--no-points", action="store_true", help="skip decode at batch 1 and 64")
    parser.add_argument("--no-prefill", action="store_true", help="skip the 2,048-token prefill measurement")
    parser.add_argument("--no-cuda-graphs", action="store_true", help="launch decode kernels one by one (for profilers)")
    parser.add_argument("--repeats", type=int, default=5, help="least number of repeats of the timed K-step region")
    parser.add_argument("--sync-scheduling", action="store_true",
                        help="read every step's tokens before the next step is planned (default: the engine's async scheduling)")
    parser.add_argument("--batch-invariant", default="off", choices=["off", "decode", "full"],
                        help="measure with the engine's bitwise-invariance modes (the default run has them off)")
    parser.add_argument("--design", default="", choices=["", "mugizen", "vivesun", "beralix", "nefipel", "pubulix", "difavik"],
                        help="measure this design beside the engine's closest other model at equal layer sizes instead of the headline")
    parser.add_argument("--design-sizes", default="s,m,moe", help="which of the sizes s, m, moe (comma-separated)")
    parser.add_argument("--design-one", default="", help=argparse.SUPPRESS)      # size:design, one model in this process
    args = parser.parse_args()

    if args.gpus != 1:
        print(f"bench.py: this engine runs on one GPU; --gpus {args.gpus} is not supported")
        return 2
    if args.warmup < 3:
        args.warmup = 3
    global CONTEXT, PAGE
    PAGE = args.page
    if args.context != CONTEXT:
        if args.context < 64 or args.context % 64:
            parser.error("--context must be a multiple of 64, at least 64")
        CONTEXT = args.context
        for _, config in SIZES.values():
            config["max_position_embeddings"] = max(config["max_position_embeddings"], CONTEXT + 2048)
    if args.impl == "reference":
        return reference_main(args)
    if args.design:
        if any(name not in DESIGN_SIZES for name in args.design_sizes.split(",")):
            parser.error(f"--design-sizes takes {sorted(DESIGN_SIZES)}")
        return design_main(args)

    import torch
    from vosti_b200 import Engine
    from vosti_b200.config import model_spec_from_config
    from vosti_b200.models import expected_weights
    from vosti_b200.weights import draw_tensors

    peaks, peak_kind = load_peaks()
    name, config = SIZES[args.size]
    config = dict(config)
    layers_full = config["num_hidden_layers"]
    if args.layers:
        config["num_hidden_layers"] = args.layers
    spec = model_spec_from_config(config)
    device = torch.device("cuda:0")
    torch.cuda.set_device(device)
    tensors = draw_tensors(expected_weights(spec), seed=0, device=device, dtype=torch.bfloat16)
    L, H = config["num_hidden_layers"], config["hidden_size"]
    nq, nkv, d, I, V = (config["num_attention_heads"], config["num_key_value_heads"], config["head_dim"],
                        config["intermediate_size"], config["vocab_size"])
    shape = {"model": name, "layers": L, "layers_full": layers_full, "hidden": H, "heads": nq, "kv_heads": nkv,
             "head_dim": d, "intermediate": I, "vocab": V}

    if args.workload == "mixed":
        num_blocks = 32 * ((3072 + 512 + PAGE) // PAGE) + 8
        engine = Engine(spec=spec, tensors=tensors, dtype="bfloat16", device="cuda:0", num_blocks=num_blocks,
                        block_size=PAGE, max_num_seqs=32, max_num_batched_tokens=4096, enable_prefix_caching=True,
                        cuda_graphs=not args.no_cuda_graphs, batch_invariant=args.batch_invariant,
                        async_scheduling=not args.sync_scheduling, consume_tensors=True)
        del tensors
        torch.cuda.empty_cache()
        mixed_run(engine, config, seed=4, requests=4)            # warm the kernels and the graphs' first shapes
        sampler = ClockSampler()
        sampler.start()
        run = mixed_run(engine, config, seed=5)
        clocks = sampler.stop()
        line = {
            "metric": f"generated tok/s, mixed continuous batch ({name})", "value": round(run["generated"] / run["wall_s"], 1),
            "unit": "tok/s", "n_gpus": 1, "steps": run["steps"], "warmup": 0,
            "ms_per_step": round(run["wall_s"] * 1e3 / max(run["steps"], 1), 4), "higher_is_better": True,
            "scaling": "weak", "vs_baseline": None, "dtype": "bf16",
            "data": "synthetic: random token ids, random-init weights", "impl": "ours",
            "config": {**shape, "global_batch": 32, "seq_len": 3072, "page_size": PAGE, "parallelism": "1 GPU",
                       "workload": "32 requests, prompts U[64,3072], 128-512 new tokens, Poisson arrivals at 16/s, "
                                   "half share a 1,024-token prefix", "peaks": peak_kind},
            "mixed": {k: (round(v, 4) if isinstance(v, float) else v) for k, v in run.items()},
            "clocks": clocks,
        }
        print(json.dumps(line))
        return 0

    max_batch = args.batch if args.no_points else max(args.batch, 64)
    tokens_per_request = CONTEXT + 2 * DECODE_STEPS + 128     # prompt, both timed regions, warm-up and slack
    num_blocks = max_batch * ((tokens_per_request + PAGE - 1) // PAGE) + 8
    engine = Engine(spec=spec, tensors=tensors, dtype="bfloat16", device="cuda:0", num_blocks=num_blocks,
                    block_size=PAGE, max_num_seqs=max_batch, max_num_batched_tokens=2 * CONTEXT,
                    enable_prefix_caching=False, cuda_graphs=not args.no_cuda_graphs,
                    batch_invariant=args.batch_invariant, async_scheduling=not args.sync_scheduling,
                    consume_tensors=True)
    del tensors
    torch.cuda.empty_cache()
    weight_bytes = engine.runner.model.weight_bytes()
    assert abs(weight_bytes - closed_form_weight_bytes(config)) <= 0.002 * weight_bytes, \
        (weight_bytes, closed_form_weight_bytes(config))
    kv_bytes_per_token = engine.runner.cache.bytes_per_token()

    prefill_ms = float("nan") if args.no_prefill else prefill_run(engine, 5, seed=11)
    main_run = decode_run(engine, args.batch, args.steps, args.warmup, seed=21, sample_clocks=True,
                          least_repeats=args.repeats)
    points = {}
    if not args.no_points:
        for batch in (1, 64):
            run = decode_run(engine, batch, max(8, args.steps // 2), 3, seed=31 + batch, least_repeats=3)
            points[f"decode_b{batch}"] = round(batch * 1e3 / run["device_ms"], 1)

    prefill_tflops = flops_of_prefill(config, CONTEXT) / (prefill_ms * 1e-3) / 1e12
    step_bytes = weight_bytes + args.batch * main_run["context"] * kv_bytes_per_token
    achieved_gbs = step_bytes / (main_run["device_ms"] * 1e-3) / 1e9

    value = args.batch * 1e3 / main_run["device_ms"]
    line = {
        "metric": f"decode tok/s at batch {args.batch} ({name}, context {CONTEXT})", "value": round(value, 1),
        "unit": "tok/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
        "ms_per_step": round(main_run["device_ms"], 4), "higher_is_better": True, "scaling": "weak",
        "vs_baseline": None, "dtype": "bf16", "data": "synthetic: random token ids, random-init weights",
        "impl": "ours",
        "config": {**shape, "global_batch": args.batch, "seq_len": CONTEXT, "page_size": PAGE, "parallelism": "1 GPU",
                   "invariance": args.batch_invariant, "scheduling": "sync" if args.sync_scheduling else "async",
                   "repeats": main_run["repeats"], "l2": "inputs larger than L2 (weights read every step)",
                   "peaks": peak_kind},
        "e2e": {"value": round(args.batch * 1e3 / main_run["wall_ms"], 1), "unit": "tok/s",
                "h2d_bytes_per_step": main_run["h2d"], "d2h_bytes_per_step": main_run["d2h"]},
        "gpu_launches": main_run["launches"],
        "clocks": main_run["clocks"],
        "prefill": {"value": round(CONTEXT * 1e3 / prefill_ms, 1), "tokens": CONTEXT, "ms": round(prefill_ms, 3),
                    "frac": round(prefill_tflops / peaks["bf16_tflops"], 4),
                    "frac_of_sustained": round(prefill_tflops / peaks.get("bf16_tflops_sustained", peaks["bf16_tflops"]), 4)},
        "roofline": {"bound": "hbm", "achieved": round(achieved_gbs, 1), "peak": peaks["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved_gbs / peaks["hbm_gbs"], 4), "bytes_per_step": int(step_bytes),
                     "weight_bytes": int(weight_bytes), "kv_bytes": int(step_bytes - weight_bytes)},
        "points": points,
    }
    print(json.dumps(line))
    return 0


if __name__ == "__main__":
    sys.exit(main())
