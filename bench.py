#!/usr/bin/env python3
"""Benchmark of janus_b200 on one B200: decode tokens per second of a
Llama-3.1-8B-shaped model with random bf16 weights (batch 8, sequences filled to
2,048 tokens of a 4,096 context), plus prefill of 2,048 tokens and decode at
batch 1 and 64.  A "step" is one decode step.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl reference]

Prints one JSON line.  `value` is timed on the device with CUDA events around K
steps of the engine's step function (index buffer copied from pinned host
memory each step, kernels replayed from a CUDA graph); `e2e` is the same metric
through `Model.generate` (host token ids in, sampled ids out each step).  Where
K steps take less than half a second the block of K steps is timed again until
half a second is covered, and the median block is reported (`config.timed_blocks`).
Both numbers follow one rule: the device idles 0.5 s after the cache is filled
(the prompt steps run at the board's power cap), then W untimed steps, then the
timed blocks.  Each step reads every weight once (15 GB, far larger than the
126 MB L2), so no L2 flush is needed between steps.  Before anything is timed,
the bfloat16 model's logits are compared with those of the true 32-bit engine on
the same weights (`checked`).

Other modes (one JSON line per item, none of them the headline): --kernels,
--prompt-lengths, --workload 1b|13b, --deterministic, --plan-check, --cpu-baseline, --float32, --design
(the Zivitar design, or with --design-model ramolix | mugedra | buludra | forisun | mibezen another one, beside the Llama decoder at equal layer
sizes: prompt and decode throughput, a step's kernels).
"""
import argparse
import json
import os
import statistics
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

# Llama-3.1-8B shape
CONFIG_8B = dict(
    architectures=["LlamaForCausalLM"], hidden_size=4096, num_hidden_layers=32, num_attention_heads=32,
    num_key_value_heads=8, head_dim=128, intermediate_size=14336, vocab_size=128256,
    max_position_embeddings=4096, rms_norm_eps=1e-5, rope_theta=500000.0,
    rope_scaling=dict(rope_type="llama3", factor=8.0, low_freq_factor=1.0, high_freq_factor=4.0,
                      original_max_position_embeddings=8192),
    tie_word_embeddings=False)
FILL = 2048          # tokens each sequence holds before decoding is timed
PREFILL_TOKENS = 2048
SETTLE_S = 0.5       # idle time after the cache is filled, before decode steps are warmed up and timed
MIN_TIMED_S = 0.5    # a timed block of K steps is repeated until this much time is covered
MAX_BLOCKS = 16
CHECK_PROMPT = 64    # tokens of the prompt whose logits are compared with the 32-bit engine before timing
BF16_LAYER_ERR = 1.1e-2   # rms error of the logits a bfloat16 layer may add, as a share of their rms (x sqrt(layers))
FALLBACK_PEAKS = dict(hbm_gbs=6650.0, bf16_tflops=1590.0, bf16_tflops_sustained=1400.0)


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        try:
            with open(path) as f:
                d = json.load(f)
            return dict(hbm_gbs=float(d["hbm_gbs"]), bf16_tflops=float(d["bf16_tflops"]),
                        bf16_tflops_sustained=float(d.get("bf16_tflops_sustained", d["bf16_tflops"])),
                        source="measured")
        except (OSError, ValueError, KeyError):
            pass
    return dict(FALLBACK_PEAKS, source="fallback")


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while a region is timed."""
    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.rows, self.proc = [], None

    def start(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", "-i", "0", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits", "-lms", "25"],
                stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.rows.append([c.strip() for c in line.split(",")])

    def stop(self):
        if self.proc is not None:
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()
        sm = [int(r[0]) for r in self.rows if len(r) >= 6 and r[0].isdigit()]
        mx = [int(r[1]) for r in self.rows if len(r) >= 6 and r[1].isdigit()]
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = [n for i, n in enumerate(names) if any(len(r) >= 6 and r[2 + i].lower() == "active" for r in self.rows)]
        return dict(sm_mhz=int(statistics.median(sm)) if sm else None, sm_max_mhz=max(mx) if mx else None,
                    reasons=reasons, samples=len(sm))


def model_numbers(cfg, layers):
    H, I, V = cfg["hidden_size"], cfg["intermediate_size"], cfg["vocab_size"]
    nh, nkv, hd = cfg["num_attention_heads"], cfg["num_key_value_heads"], cfg["head_dim"]
    per_layer = H * (nh + 2 * nkv) * hd + nh * hd * H + 3 * H * I          # matrix elements
    return dict(layer_params=per_layer, head_params=V * H, kv_bytes_per_token=2 * nkv * hd * 2 * layers,
                norm_bytes=(2 * layers + 1) * H * 2)


def decode_bytes(cfg, layers, batch, ctx):
    n = model_numbers(cfg, layers)
    return 2 * (layers * n["layer_params"] + n["head_params"]) + n["norm_bytes"] + batch * ctx * n["kv_bytes_per_token"]


def prefill_flops(cfg, layers, T):
    n = model_numbers(cfg, layers)
    linear = 2 * T * layers * n["layer_params"] + 2 * n["head_params"]      # the head runs on one row
    attention = layers * 4 * cfg["num_attention_heads"] * cfg["head_dim"] * T * (T + 1) // 2
    return linear + attention


def rms_err(got, ref):
    import numpy as np
    got, ref = got.astype(np.float64), ref.astype(np.float64)
    if not np.isfinite(got).all():
        return float("inf")
    return float(np.sqrt(((got - ref) ** 2).mean()) / np.sqrt((ref ** 2).mean()))


def check_against_float32(cfg, layers, prompt):
    """Logits of the bfloat16 model at four rows of a 64-token prompt against the true 32-bit engine on the
    same weights (the benchmark's: seed 2, stored as bfloat16).  Returns (ok, rms error, bound)."""
    import torch

    import janus_b200
    from janus_b200.engine import StepEntry
    rows = [0, CHECK_PROMPT // 3, 2 * CHECK_PROMPT // 3, CHECK_PROMPT - 1]
    outs = {}
    for dtype in ("float32", "bfloat16"):
        model = janus_b200.load_random(cfg, seed=2, dtype=dtype, max_tokens=128, max_slots=1, norm_std=0.0,
                                       stored_dtype="bfloat16")
        outs[dtype] = model.step([StepEntry(model.alloc_slot(), prompt[:CHECK_PROMPT], rows)]).cpu().numpy()
        model.check()
        del model
        torch.cuda.empty_cache()
    err, bound = rms_err(outs["bfloat16"], outs["float32"]), BF16_LAYER_ERR * layers ** 0.5
    return err < bound, err, bound


def run_ours(args):
    import torch

    import janus_b200
    from janus_b200.engine import StepEntry
    from janus_b200.kernels import ops

    if args.deterministic:
        ops.set_deterministic(True)
    layers = args.layers or CONFIG_8B["num_hidden_layers"]
    cfg = dict(CONFIG_8B, num_hidden_layers=layers)
    K, W = args.steps, args.warmup
    batches = [1, 8, 64] if not args.quick else [args.batch]
    max_b = max(batches)
    g = torch.Generator().manual_seed(0)
    V = cfg["vocab_size"]

    def tokens(n):
        return torch.randint(0, V, (n,), generator=g).tolist()

    prompt = tokens(PREFILL_TOKENS)
    checked, check_err, check_bound = (None, None, None)
    if not args.no_check:
        checked, check_err, check_bound = check_against_float32(cfg, layers, prompt)
        if not checked:
            print(f"bench: the bfloat16 logits differ from the 32-bit engine's by {check_err:.4f} rms "
                  f"(bound {check_bound:.4f}); nothing is timed", file=sys.stderr)
            return 1

    max_steps = W + MAX_BLOCKS * K + 8
    per_seq = FILL + 2 * max_steps + 128
    model = janus_b200.load_random(cfg, seed=2, dtype="bfloat16", max_tokens=max_b * (per_seq + 64),
                                   max_slots=max_b, norm_std=0.0)
    eng = model.engine
    dev = model.device

    def timed(fn, reps):
        start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize(dev)
        start.record()
        for _ in range(reps):
            fn()
        end.record()
        torch.cuda.synchronize(dev)
        return start.elapsed_time(end) / reps

    # ---- prefill of 2,048 tokens ------------------------------------------------
    def one_prefill():
        s = eng.alloc_slot()
        eng.step([StepEntry(s, prompt, (PREFILL_TOKENS - 1,))])
        eng.free_slot(s)

    for _ in range(3):
        one_prefill()
    prefill_ms = timed(one_prefill, 5)
    pk = peaks()
    flops = prefill_flops(cfg, layers, PREFILL_TOKENS)
    prefill = dict(value=round(PREFILL_TOKENS / prefill_ms * 1e3, 1), tokens=PREFILL_TOKENS, ms=round(prefill_ms, 3),
                   frac=round(flops / (prefill_ms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4),
                   frac_of_sustained=round(flops / (prefill_ms * 1e-3) / (pk["bf16_tflops_sustained"] * 1e12), 4))

    # ---- decode at each batch size ----------------------------------------------
    torch.cuda.profiler.start()          # for `ncu --profile-from-start off`: the decode steps from here on
    results, launches = {}, {}
    clocks = None
    for B in batches:
        slots = [eng.alloc_slot() for _ in range(B)]
        for i in range(0, B, 8):                                   # fill the sequences, 8 prompts a step
            eng.step([StepEntry(s, tokens(FILL), ()) for s in slots[i:i + 8]])
        pool = [[int(t) for t in tokens(B)] for _ in range(64)]
        turn = [0]
        # The fill ran at the board's power cap; the SM clocks take some 150 ms to come back after it
        # (measured: the first ~30 decode steps after a 16k-token prefill take 4.4 - 5.1 ms instead of 3.6).
        # Decoding is timed in its steady state, so the device idles briefly first.
        torch.cuda.synchronize(dev)
        time.sleep(SETTLE_S)

        def one_step():
            row = pool[turn[0] % len(pool)]
            turn[0] += 1
            eng.step([StepEntry(s, (t,), (0,)) for s, t in zip(slots, row)], borrow=True)

        for _ in range(W):
            one_step()
        per_step_launches = eng.last_graph_launches
        sampler = ClockSampler() if B == args.batch else None
        if sampler:
            sampler.start()
        blocks, covered = [], 0.0
        while len(blocks) < MAX_BLOCKS and (not blocks or covered < MIN_TIMED_S):
            blocks.append(timed(one_step, K))
            covered += blocks[-1] * K * 1e-3
        if sampler:
            clocks = sampler.stop()
        ops.check_kernel_status(dev)
        order = sorted(range(len(blocks)), key=lambda i: blocks[i])
        mid = order[(len(blocks) - 1) // 2]                         # the median block (the lower of two)
        ms = blocks[mid]
        results[B] = dict(ms=ms, tok_s=B / ms * 1e3, blocks=len(blocks), ctx=FILL + W + mid * K + K // 2,
                          spread=round((max(blocks) - min(blocks)) / ms, 4))
        launches[B] = per_step_launches * K
        for s in slots:
            eng.free_slot(s)

    # ---- end to end through the public entry point ----------------------------------
    B = args.batch
    n_blocks = results[B]["blocks"]
    prompts = [tokens(FILL) for _ in range(B)]
    model.generate(prompts, max_tokens=W + 2, ignore_eos=True)                       # warm-up (graphs are captured)
    # One generation of W + n_blocks * K + 1 tokens under the same rule as above: when the prefill's tokens
    # arrive the host idles 0.5 s, then W untimed decode steps, then blocks of K steps on the host clock,
    # from the arrival of one step's tokens to the arrival of the tokens K steps later: each step with its
    # index buffer copied from pinned host memory and its sampled tokens read back.  The median block counts.
    arrivals = []

    def on_token(request, token):
        if request == 0:
            if not arrivals:
                torch.cuda.synchronize(dev)
                time.sleep(SETTLE_S)
            arrivals.append(time.perf_counter())
        return True

    model.generate(prompts, max_tokens=W + n_blocks * K + 1, ignore_eos=True, callback=on_token)
    # arrivals[0] is the prefill's token; arrivals[i] that of decode step i
    e2e_blocks = sorted(B * K / (arrivals[W + (i + 1) * K] - arrivals[W + i * K]) for i in range(n_blocks))
    e2e_tok_s = e2e_blocks[(n_blocks - 1) // 2]

    head = results[args.batch]
    nbytes = decode_bytes(cfg, layers, args.batch, head["ctx"])
    achieved = nbytes / (head["ms"] * 1e-3) / 1e9
    out = {
        "metric": "decode tok/s @ batch 8 (Llama-3-8B shape, bf16, ctx 4096, sequences at 2048)",
        "value": round(head["tok_s"], 1), "unit": "tokens/s", "n_gpus": 1, "steps": K, "warmup": W,
        "ms_per_step": round(head["ms"], 4), "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic token ids, random-init weights (seed 2)", "impl": "janus_b200",
        "config": {
            "model": "Llama-3.1-8B shape", "layers": layers, "layers_of_config": CONFIG_8B["num_hidden_layers"],
            "hidden": cfg["hidden_size"], "heads": cfg["num_attention_heads"], "kv_heads": cfg["num_key_value_heads"],
            "head_dim": cfg["head_dim"], "intermediate": cfg["intermediate_size"], "vocab": cfg["vocab_size"],
            "global_batch": args.batch, "seq_len": 4096, "filled_to": FILL, "prefill_tokens": PREFILL_TOKENS,
            "parallelism": "single GPU", "l2": "inputs larger than L2 (15 GB of weights per step)",
            "peaks": pk["source"], "timed_blocks": head["blocks"], "block_spread": head["spread"],
            "settle_s": SETTLE_S, "deterministic": bool(args.deterministic),
        },
        "e2e": {"value": round(e2e_tok_s, 1), "unit": "tokens/s",
                "h2d_bytes_per_step": eng.last_step_h2d_bytes + 3 * 4 * B, "d2h_bytes_per_step": 4 * B,
                "steps": K, "warmup": W, "blocks": n_blocks},
        "gpu_launches": launches[args.batch],
        "prefill": prefill,
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4)},
        "points": {f"decode_b{b}": round(r["tok_s"], 1) for b, r in results.items() if b != args.batch},
        "point_fracs": {f"decode_b{b}": round(decode_bytes(cfg, layers, b, r["ctx"]) / (r["ms"] * 1e-3) / 1e9
                                              / pk["hbm_gbs"], 4) for b, r in results.items() if b != args.batch},
        "checked": checked,
        "check": None if checked is None else {"rms_err_vs_float32": round(check_err, 5), "bound": round(check_bound, 5),
                                               "rows": 4, "prompt_tokens": CHECK_PROMPT},
        "clocks": clocks,
    }
    print(json.dumps(out))
    return 0


# whole workloads through the public entry point
WORKLOADS = {
    "1b": dict(
        config=dict(architectures=["LlamaForCausalLM"], hidden_size=2048, num_hidden_layers=16, num_attention_heads=32,
                    num_key_value_heads=8, head_dim=64, intermediate_size=8192, vocab_size=128256,
                    max_position_embeddings=2048, rms_norm_eps=1e-5, rope_theta=500000.0,
                    rope_scaling=dict(rope_type="llama3", factor=32.0, low_freq_factor=1.0, high_freq_factor=4.0,
                                      original_max_position_embeddings=8192),
                    tie_word_embeddings=True),
        seed=3, batch=64, prompt_range=(16, 1024), max_new=256, context=2048),
    "13b": dict(
        config=dict(architectures=["LlamaForCausalLM"], hidden_size=5120, num_hidden_layers=40, num_attention_heads=40,
                    num_key_value_heads=40, head_dim=128, intermediate_size=13824, vocab_size=32000,
                    max_position_embeddings=4096, rms_norm_eps=1e-5, rope_theta=10000.0, rope_scaling=None,
                    tie_word_embeddings=False),
        seed=4, batch=16, prompt_range=(128, 3072), max_new=4096, context=4096),
}


def run_workload(name):
    """A whole workload of BASELINE.json (1B: 64 sequences, prompts U[16,1024], 256 new tokens each;
    13B: batch 16, prompts U[128,3072], decoding until 4,096 positions) through Model.generate."""
    import torch

    import janus_b200
    w = WORKLOADS[name]
    g = torch.Generator().manual_seed(w["seed"])
    lo, hi = w["prompt_range"]
    lens = torch.randint(lo, hi + 1, (w["batch"],), generator=g).tolist()
    V = w["config"]["vocab_size"]
    prompts = [torch.randint(0, V, (n,), generator=g).tolist() for n in lens]
    room = sum((min(n + w["max_new"], w["context"]) + 63) // 64 * 64 for n in lens)
    model = janus_b200.load_random(w["config"], seed=w["seed"], dtype="bfloat16", max_tokens=room + 64 * w["batch"],
                                   max_slots=w["batch"], max_seq_len=w["context"], norm_std=0.0)
    model.generate([p[:32] for p in prompts[:w["batch"]]], max_tokens=4, ignore_eos=True)      # warm-up
    torch.cuda.synchronize()
    torch.cuda.profiler.start()          # for `ncu --profile-from-start off`: nothing before this is captured
    t0 = time.perf_counter()
    out, stats = model.generate(prompts, max_tokens=w["max_new"], ignore_eos=True)
    torch.cuda.synchronize()
    wall = time.perf_counter() - t0
    torch.cuda.profiler.stop()
    new_tokens = sum(len(o) for o in out)
    # what the decode steps had to read: every weight once per step, and the cached keys and values of the
    # sequences that were live at the step (request r's j-th decode step reads prompt + j tokens)
    cfg, L = w["config"], w["config"]["num_hidden_layers"]
    n = model_numbers(cfg, L)
    weight_bytes = 2 * (L * n["layer_params"] + n["head_params"]) + n["norm_bytes"]
    kv_tokens = sum(sum(range(ln + 1, ln + len(o))) for ln, o in zip(lens, out))
    step_bytes = stats.decode_steps * weight_bytes + kv_tokens * n["kv_bytes_per_token"]
    pk = peaks()
    achieved = step_bytes / (stats.decode_ms * 1e-3) / 1e9 if stats.decode_ms > 0 else 0.0
    print(json.dumps({
        "impl": "janus_b200", "workload": name, "metric": "generated tokens/s, whole workload through Model.generate",
        "value": round(new_tokens / wall, 1), "unit": "tokens/s", "wall_s": round(wall, 3),
        "prompt_tokens": sum(lens), "new_tokens": new_tokens, "decode_steps": stats.decode_steps,
        "prefill_tokens_per_s": round(stats.prefill_tokens_per_s, 1),
        "decode_tokens_per_s": round(stats.decode_tokens_per_s, 1), "dtype": "bf16",
        "decode_ms_per_step": round(stats.decode_ms / max(1, stats.decode_steps), 4),
        "graph_captures": stats.graph_captures,
        "roofline": {"bound": "hbm", "what": "decode steps: weights once per step + live sequences' cache",
                     "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4), "peaks": pk["source"]},
        "data": f"synthetic token ids, random-init weights (seed {w['seed']})",
        "config": {"batch": w["batch"], "prompt_lengths": f"U[{lo},{hi}]", "context": w["context"],
                   "layers": w["config"]["num_hidden_layers"], "hidden": w["config"]["hidden_size"],
                   "heads": w["config"]["num_attention_heads"], "kv_heads": w["config"]["num_key_value_heads"],
                   "head_dim": w["config"]["head_dim"], "intermediate": w["config"]["intermediate_size"],
                   "vocab": V}}))


PROMPT_STEPS = "1x96,1x128,1x256,1x384,1x512,1x768,1x1024,1x1536,1x2048,1x4096,4x256,8x100"


def run_prompt_lengths(layers, which):
    """Prompt steps of 96 to 4,096 tokens at the 8B layer sizes (fewer layers, named in each line): device
    time of `Model.step` with the logits of the last token, median of 5 after 3 warm-ups.  The device idles
    50 ms before each measured step (JANUS_BENCH_GAP_S; long steps run into the power cap, and the clocks need
    the pause to come back; steps of up to 256 tokens measure 5 to 8 % faster back to back).  One JSON line per
    length; nothing here is the headline."""
    import torch

    import janus_b200
    from janus_b200.engine import StepEntry
    cases = [tuple(int(v) for v in item.split("x")) for item in which.split(",")]
    cfg = dict(CONFIG_8B, num_hidden_layers=layers, max_position_embeddings=max(8192, max(t for _, t in cases)))
    model = janus_b200.load_random(cfg, seed=2, dtype="bfloat16", max_tokens=max(16384, max(s * t for s, t in cases)),
                                   max_slots=16, norm_std=0.0)
    torch.cuda.profiler.start()          # for `ncu --profile-from-start off`: nothing of the weights' set-up is captured
    g = torch.Generator().manual_seed(0)
    pk = peaks()
    for seqs, T in cases:
        times = []
        for _ in range(8):
            slots = [model.alloc_slot() for _ in range(seqs)]
            entries = [StepEntry(s, torch.randint(0, cfg["vocab_size"], (T,), generator=g).tolist(), [T - 1])
                       for s in slots]
            torch.cuda.synchronize()
            time.sleep(float(os.environ.get("JANUS_BENCH_GAP_S", "0.05")))
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            model.step(entries)
            b.record()
            torch.cuda.synchronize()
            times.append(a.elapsed_time(b))
            for s in slots:
                model.free_slot(s)
        ms = sorted(times[3:])[2]
        flops = layers * seqs * (2 * T * layer_weight_elems(cfg) + 2 * 2 * cfg["num_attention_heads"] * cfg["head_dim"]
                                 * T * (T + 1) / 2)
        print(json.dumps({"prompt_step": f"{seqs} x {T} tokens", "layers": layers, "layers_of_config": 32,
                          "ms": round(ms, 3), "tokens_per_s": round(seqs * T / ms * 1e3),
                          "layer_flops_frac": round(flops / (ms * 1e-3) / (pk["bf16_tflops"] * 1e12), 3),
                          "peaks": pk.get("source", "fallback")}), flush=True)
    model.check()


def run_float32(layers):
    """The true 32-bit path (the oracle's, not the serving one) at the 8B layer sizes through Model.generate:
    8 prompts of 2,048 tokens, then 16 tokens each, and one sequence alone.  One JSON line; nothing here is the
    headline."""
    import torch

    import janus_b200
    cfg = dict(CONFIG_8B, num_hidden_layers=layers)
    model = janus_b200.load_random(cfg, seed=2, dtype="float32", max_tokens=8 * 2304, max_slots=8, norm_std=0.0,
                                   stored_dtype="bfloat16")
    g = torch.Generator().manual_seed(0)
    prompts = [torch.randint(0, cfg["vocab_size"], (2048,), generator=g).tolist() for _ in range(8)]
    model.generate(prompts, max_tokens=2, ignore_eos=True)            # first touch of the workspaces
    _, st8 = model.generate(prompts, max_tokens=16, ignore_eos=True)
    _, st1 = model.generate(prompts[:1], max_tokens=16, ignore_eos=True)
    n = model_numbers(cfg, layers)
    weight_bytes = 4 * (layers * n["layer_params"] + n["head_params"])
    ms8 = st8.decode_ms / st8.decode_steps
    print(json.dumps({"impl": "janus_b200", "dtype": "float32", "layers": layers, "layers_of_config": 32,
                      "decode_b8_tokens_per_s": round(st8.decode_tokens_per_s, 1), "decode_b8_ms_per_step": round(ms8, 2),
                      "decode_b1_tokens_per_s": round(st1.decode_tokens_per_s, 1),
                      "prefill_tokens_per_s": round(st8.prefill_tokens_per_s),
                      "weights_GBps_b8": round(weight_bytes / ms8 / 1e6, 1),
                      "frac_of_hbm_b8": round(weight_bytes / ms8 / 1e6 / peaks()["hbm_gbs"], 3)}), flush=True)


def layer_weight_elems(cfg):
    hd = cfg["head_dim"]
    qkv = (cfg["num_attention_heads"] + 2 * cfg["num_key_value_heads"]) * hd * cfg["hidden_size"]
    o = cfg["num_attention_heads"] * hd * cfg["hidden_size"]
    return qkv + o + 3 * cfg["intermediate_size"] * cfg["hidden_size"]


KERNEL_SHAPES = {   # hidden, heads, kv heads, head size, intermediate, vocabulary
    "8b": (4096, 32, 8, 128, 14336, 128256),
    "1b": (2048, 32, 8, 64, 8192, 128256),
    "13b": (5120, 40, 40, 128, 13824, 32000),
}


def run_kernels(contexts=None, shape="8b", head_sizes=None):
    """The step's hot kernels alone at the 8B layer shapes, for the roofline figures under profiles/:
    each is captured 24 times into one CUDA graph (as the engine runs them: back to back, programmatic
    dependent launch) over several copies of its weights or cache, so that every launch reads from DRAM,
    and timed with CUDA events around 5 replays.  One line per kernel; nothing here is the headline.
    With `contexts` (key counts), decode attention alone at those contexts, for 1, 8 and 64 sequences.
    With `head_sizes`, prompt attention alone at those head sizes (the shape's heads; 2,048 tokens, or one
    prompt of each of `contexts`) on both of its kernels: tcgen05 (head sizes up to 128) and mma.sync."""
    import math

    import torch

    from janus_b200.kernels import ops
    dev = "cuda:0"
    H, NH, NKV, HD, I, V = KERNEL_SHAPES[shape]

    def timed(fn, reps=24):
        for _ in range(3):
            fn()
        torch.cuda.synchronize()
        time.sleep(SETTLE_S)              # the clocks come back from the power cap of the kernel before
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g):
            for _ in range(reps):
                fn()
        g.replay()
        torch.cuda.synchronize()
        start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        start.record()
        for _ in range(5):
            g.replay()
        end.record()
        torch.cuda.synchronize()
        return start.elapsed_time(end) / (5 * reps) * 1e3          # microseconds per launch

    class Scratch:
        def __init__(self):
            self.buffers = {}

        def get(self, name, shape, dtype):
            n = math.prod(shape)
            if name not in self.buffers or self.buffers[name].numel() < n:
                self.buffers[name] = torch.empty(n, dtype=dtype, device=dev)
            return self.buffers[name][:n].view(*shape)

    def product(name, T, N, K, mode, copies=6):
        rows = 2 * N if mode == "swiglu" else N
        def weight():
            w = (torch.randn(rows, K, device=dev) * 0.02).to(torch.bfloat16)
            return ops.pack_gated(w[:N].contiguous(), w[N:].contiguous()) if mode == "swiglu" else ops.pack_weight(w)

        ws = [weight() for _ in range(copies)]
        x = torch.randn(T, K, device=dev).to(torch.bfloat16)
        y = torch.zeros(T, N, device=dev, dtype=torch.bfloat16 if mode == "swiglu" else torch.float32)
        turn = [0]
        # a stored product of few tokens runs as the engine runs it: scratch cleared, slices of K added
        as_add = mode == "store" and T <= 64 and ops.split_k_for(T, N, K) > 1

        def fn():
            w = ws[turn[0] % copies]
            turn[0] += 1
            if as_add:
                ops.zero_f32(y)
                ops.gemm_bf16(x, w, y, mode="add")
            else:
                ops.gemm_bf16(x, w, y, mode=mode)

        us = timed(fn)
        print(json.dumps({"kernel": f"product {name}", "tokens": T, "us": round(us, 1),
                          "weights_GBps": round(rows * K * 2 / us / 1e3, 1),
                          "TFLOPs": round(2 * T * rows * K / us / 1e6, 1)}), flush=True)

    if not contexts and not head_sizes:
        for T in (8, 64, 2048):
            product("qkv", T, (NH + 2 * NKV) * HD, H, "store")
            product("o (add)", T, H, NH * HD, "add")
            product("gate_up (SiLU gate)", T, I, H, "swiglu")
            product("down (add)", T, H, I, "add")
        product("lm_head", 8, V, H, "store", copies=3)
        # the RMS norm (float32 rows in, bfloat16 out) at a decode step's and at prompts' row counts
        gamma = torch.ones(H, device=dev, dtype=torch.bfloat16)
        for T in (8, 2048, 16384):
            xs = [torch.randn(T, H, device=dev) for _ in range(4)]
            y = torch.empty(T, H, device=dev, dtype=torch.bfloat16)
            turn = [0]

            def norm():
                ops.rmsnorm(xs[turn[0] % 4], gamma, 1e-5, y)
                turn[0] += 1

            us = timed(norm)
            print(json.dumps({"kernel": "rmsnorm", "rows": T, "us": round(us, 1),
                              "GBps": round(T * H * 6 / us / 1e3, 1)}), flush=True)
        # the sampling kernel over a decode step's logits (8 rows of the vocabulary), option by option
        from janus_b200.sampling import DeviceSampler, SamplerConfig
        logits = torch.randn(8, V, device=dev) * 3
        rows = torch.arange(8, device=dev, dtype=torch.int32)
        for name, kw in (("greedy", dict(temperature=0.0)),
                         ("greedy, repetition penalty 1.15", dict(temperature=0.0, repetition_penalty=1.15)),
                         ("temperature 0.8", dict(temperature=0.8)),
                         ("temperature 0.8, top-k 50", dict(temperature=0.8, top_k=50)),
                         ("temperature 0.8, top-p 0.9", dict(temperature=0.8, top_p=0.9)),
                         ("temperature 0.8, top-k 50, top-p 0.9, repetition penalty 1.15",
                          dict(temperature=0.8, top_k=50, top_p=0.9, repetition_penalty=1.15))):
            sampler = DeviceSampler(SamplerConfig(max_tokens=8, **kw), V, 8, 0, torch.device(dev))
            us = timed(lambda: sampler.sample(logits, rows, rows, rows))
            print(json.dumps({"kernel": f"sample ({name})", "rows": 8, "vocabulary": V, "us": round(us, 1)}),
                  flush=True)

    cases = [(b, c) for c in contexts for b in (1, 8, 64) if b * c <= 1 << 21] if contexts else ((1, 2080), (8, 2080), (64, 2080))
    if head_sizes:
        cases = ()
    for B, ctx in cases:
        pages = (ctx + 63) // 64
        n_pages = B * pages
        copies = max(1, min(8, int(3e9 // (n_pages * NKV * 64 * HD * 4))))
        kcs = [torch.randn(n_pages, NKV, 64, HD, device=dev).to(torch.bfloat16) for _ in range(copies)]
        vcs = [torch.randn(n_pages, NKV, 64, HD, device=dev).to(torch.bfloat16) for _ in range(copies)]
        table = torch.arange(n_pages, device=dev, dtype=torch.int32).view(B, pages)
        kv_len = torch.full((B,), ctx, device=dev, dtype=torch.int32)
        q = torch.randn(B, NH * HD, device=dev).to(torch.bfloat16)
        out = torch.empty_like(q)
        ws, turn = Scratch(), [0]
        cap = 1 << (pages - 1).bit_length()                          # the engine's graphs are keyed by this bound

        def fn():
            i = turn[0] % copies
            turn[0] += 1
            ops.attention_bf16_decode(q, kcs[i], vcs[i], out, table, kv_len, NH, NKV, HD, 64, 0, 1 / math.sqrt(HD),
                                      ws, cap * 64)

        us = timed(fn)
        print(json.dumps({"kernel": "decode attention + combine", "sequences": B, "keys": ctx,
                          "splits": ops.decode_splits_for(B, NKV * ((NH // NKV + 15) // 16), cap * 64, 64, HD), "us": round(us, 1),
                          "kv_GBps": round(B * ctx * NKV * HD * 4 / us / 1e3, 1)}), flush=True)

    for hd, L in ((h, c) for h in head_sizes or () for c in contexts or (2048,)):
        B = 1
        pages = (L + 63) // 64
        kc = torch.randn(B * pages, NKV, 64, hd, device=dev).to(torch.bfloat16)
        vc = torch.randn_like(kc)
        table = torch.arange(B * pages, device=dev, dtype=torch.int32).view(B, pages)
        q = torch.randn(B * L, NH * hd, device=dev).to(torch.bfloat16)
        out = torch.empty_like(q)
        q_start = torch.arange(B + 1, device=dev, dtype=torch.int32) * L
        kv_len = torch.full((B,), L, device=dev, dtype=torch.int32)
        faces = [("mma.sync", ops.attention_bf16_prefill)]
        if ops.attention_tc_supported(NH, NKV, hd):
            faces.insert(0, ("tcgen05", ops.attention_tc_prefill))
        for name, face in faces:
            if name == "mma.sync" and L > 8192:
                continue
            us = timed(lambda: face(q, kc, vc, out, table, q_start, kv_len, B, L, NH, NKV, hd, 64, 0,
                                    1 / math.sqrt(hd)), reps=6 if L <= 8192 else 2)
            print(json.dumps({"kernel": f"prefill attention ({name})", "head_size": hd, "tokens": L,
                              "us": round(us, 1),
                              "TFLOPs": round(B * 4 * NH * hd * L * (L + 1) / 2 / us / 1e6, 1)}), flush=True)
    for B, L in (() if contexts or head_sizes else ((1, 2048), (1, 8192))):
        pages = (L + 63) // 64
        kc = torch.randn(B * pages, NKV, 64, HD, device=dev).to(torch.bfloat16)
        vc = torch.randn_like(kc)
        table = torch.arange(B * pages, device=dev, dtype=torch.int32).view(B, pages)
        q = torch.randn(B * L, NH * HD, device=dev).to(torch.bfloat16)
        out = torch.empty_like(q)
        q_start = torch.arange(B + 1, device=dev, dtype=torch.int32) * L
        kv_len = torch.full((B,), L, device=dev, dtype=torch.int32)
        us = timed(lambda: ops.attention_tc_prefill(q, kc, vc, out, table, q_start, kv_len, B, L, NH, NKV, HD, 64, 0,
                                                    1 / math.sqrt(HD)), reps=6)
        print(json.dumps({"kernel": "prefill attention (tcgen05)", "tokens": L, "us": round(us, 1),
                          "TFLOPs": round(B * 4 * NH * HD * L * (L + 1) / 2 / us / 1e6, 1)}), flush=True)
    ops.check_kernel_status(torch.device(dev))


DESIGN_SIZES = {
    # name: width, feed-forward, heads, key/value heads, window; four layers each: one lightning mixer, three
    # differential attention mixers (key size 64 per map, value size 128), two residual streams
    "2k": dict(width=2048, ff=8192, heads=16, kv_heads=4, window=1024, vocab=32000),
    "4k": dict(width=4096, ff=14336, heads=32, kv_heads=8, window=2048, vocab=32000),
}


def zivitar_config(width, ff, heads, kv_heads, window, vocab):
    attention = dict(type="attention", mlp=dict(kind="dense", ff=ff, limit=7.0),
                     mixer=dict(heads=heads, kv_heads=kv_heads, dim=64, vdim=128, scale=0.125, diff=0.5, conv=4,
                                mask=dict(size=window, keep_first=4),
                                rot=dict(dims=32, base=10000.0, scaling=dict(factor=4.0, original=4096, fast=32.0, slow=1.0))))
    lightning = dict(type="lightning", mlp=dict(kind="dense", ff=ff, limit=7.0),
                     mixer=dict(heads=heads, dim=128, vdim=128, decay=[1.0 - 2.0 ** (-5 - 3 * h / heads) for h in range(heads)]))
    return dict(architecture="Zivitar", vocab=vocab, width=width, norm=dict(eps=1e-5), streams=2, logit_scale=1.0,
                logit_softcap=30.0, layers=[lightning, attention, attention, attention])


def ramolix_config(width, ff, heads, kv_heads, window, vocab):
    """Four layers at the size's width: two state-space mixers (inner width twice the model's, heads of 64 values,
    128 state rows, one group, four taps), sliding-window attention whose values are its keys (head size 128, half
    of it rotated) and latent attention (128 per head, latents of 256), each with a GELU-gated feed-forward."""
    mlp = dict(kind="dense", ff=ff)
    mamba = dict(type="mamba2", mlp=mlp, mixer=dict(heads=2 * width // 64, vdim=64, state=128, groups=1, conv=4, norm_groups=1))
    attention = dict(type="attention", mlp=mlp,
                     mixer=dict(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, scale=128 ** -0.5, mask=dict(size=window),
                                rot=dict(dims=64, base=10000.0, scaling=dict(factor=4.0, low=1.0, high=4.0, original=4096))))
    latent = dict(type="latent_attention", mlp=mlp, mixer=dict(heads=heads, dim=128, vdim=128, kv_rank=256, scale=128 ** -0.5))
    return dict(architecture="Ramolix", vocab=vocab, width=width, norm=dict(eps=1e-5), embedding=dict(scale=width ** 0.5),
                residual_mult=0.7, layers=[mamba, attention, mamba, latent])


def llama_like(width, ff, heads, kv_heads, window, vocab):
    return dict(architectures=["LlamaForCausalLM"], hidden_size=width, num_hidden_layers=4, num_attention_heads=heads,
                num_key_value_heads=kv_heads, head_dim=128, intermediate_size=ff, vocab_size=vocab,
                max_position_embeddings=16384, rms_norm_eps=1e-5, rope_theta=10000.0, rope_scaling=None,
                tie_word_embeddings=False)


def mugedra_config(width, ff, heads, kv_heads, window, vocab):
    """Three layers at the size's width of which the middle one runs twice (four layer runs): capped attention in
    chunks of the size's window (head size 128, half of it rotated) beside a gated delta rule (as many heads of 128
    by 128 state, four taps), and eight experts of half the size's feed-forward each of which a token uses two (the
    dense feed-forward's products per token)."""
    layer = dict(type="parallel",
                 mixer=dict(left=dict(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, scale=128 ** -0.5, softcap=50.0,
                                      mask=dict(size=window),
                                      rot=dict(dims=64, base=10000.0, scaling=dict(factor=4.0, original=4096, fast=32.0, slow=1.0))),
                            right=dict(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, conv=4)),
                 mlp=dict(kind="moe", expert=dict(ff=ff // 2), router=dict(experts=8, top=2)))
    return dict(architecture="Mugedra", vocab=vocab, width=width, norm=dict(eps=1e-5), loop=dict(start=1, stop=2, times=2),
                layers=[layer, layer, layer])


def buludra_config(width, ff, heads, kv_heads, window, vocab):
    """Four layers at the size's width: sink attention (head size 128, half of it rotated) beside a matrix memory with
    exponential gates (as many heads of 128 by 128 state) with a dense feed-forward; attention with normed heads and a
    query temperature with experts; gated linear attention (as many heads of 128 by 128 state, decays of rank 64)
    with a dense feed-forward; the two mixers side by side again with experts.  Eight experts of half the size's
    feed-forward each in four groups of which two are kept, two experts a token (the dense feed-forward's products
    per token), and a shared expert of a quarter of it."""
    side = dict(left=dict(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, scale=0.5 * 128 ** -0.5,
                          rot=dict(dims=64, base=10000.0)),
                right=dict(heads=heads, dim=128, vdim=128, gate_cap=15.0), left_scale=0.8, right_scale=0.9)
    experts = dict(kind="moe", expert=dict(ff=ff // 2), router=dict(experts=8, top=2, groups=dict(count=4, keep=2)),
                   shared=dict(ff=ff // 4))
    dense = dict(kind="dense", ff=ff)
    return dict(architecture="Buludra", vocab=vocab, width=width, norm=dict(eps=1e-5), logit_softcap=30.0,
                layers=[dict(type="parallel", mixer=side, mlp=dense),
                        dict(type="attention", mlp=experts,
                             mixer=dict(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, scale=128 ** -0.5,
                                        q_temp=dict(coef=0.1, every=1024))),
                        dict(type="gla", mlp=dense, mixer=dict(heads=heads, dim=128, vdim=128, tau=16.0, rank=64)),
                        dict(type="parallel", mixer=side, mlp=experts)])


def forisun_config(width, ff, heads, kv_heads, window, vocab):
    """Four layers at the size's width of latent attention with an output gate (128 unrotated and 64 rotated numbers per
    query, values of 128, latents of 512, so cached rows of 576 numbers), the last one over the third's rows; the first
    with a dense feed-forward (one matrix up, no gate), the others with eight experts of half the size's feed-forward
    each of which a token uses two (the gated dense feed-forward's products per token)."""
    mixer = dict(heads=heads, dim=128, rot_dim=64, vdim=128, kv_rank=512, scale=192 ** -0.5,
                 rot=dict(dims=64, base=10000.0, scaling=dict(factor=4.0, original=4096, fast=32.0, slow=1.0)))
    dense = dict(kind="dense", ff=ff)
    experts = dict(kind="moe", expert=dict(ff=ff // 2), router=dict(experts=8, top=2, scale=1.5))
    kind = "latent_attention"
    return dict(architecture="Forisun", vocab=vocab, width=width, norm=dict(eps=1e-5), embedding=dict(scale=width ** 0.5),
                layers=[dict(type=kind, mixer=mixer, mlp=dense), dict(type=kind, mixer=mixer, mlp=experts),
                        dict(type=kind, mixer=mixer, mlp=experts), dict(type=kind, mixer=dict(mixer, kv_from=2), mlp=experts)])


def mibezen_config(width, ff, heads, kv_heads, window, vocab):
    """Four layers at the size's width: latent attention as in `forisun_config`, its queries by way of a latent of three
    quarters of the width, and grouped-query attention with a distance bias, learned sinks and mixed values in chunks of four
    times the size's window (heads of 128, values of 128; a decode step at 2,048 keys sees them all), each kind once with a dense feed-forward (squared relu, one matrix up) and
    once with eight experts of half the size's feed-forward of which a token uses two."""
    latent = dict(heads=heads, dim=128, rot_dim=64, vdim=128, q_rank=width * 3 // 4, kv_rank=512, scale=192 ** -0.5,
                  rot=dict(dims=64, base=10000.0, scaling=dict(factor=4.0, original=4096, fast=32.0, slow=1.0)))
    chunked = dict(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, scale=128 ** -0.5, mask=dict(size=4 * window), v_mix=True)
    dense = dict(kind="dense", ff=ff)
    experts = dict(kind="moe", expert=dict(ff=ff // 2), router=dict(experts=8, top=2))
    return dict(architecture="Mibezen", vocab=vocab, width=width, norm=dict(eps=1e-6), logit_softcap=15.0,
                layers=[dict(type="latent_attention", mixer=latent, mlp=dense), dict(type="attention", mixer=chunked, mlp=experts),
                        dict(type="attention", mixer=chunked, mlp=dense), dict(type="latent_attention", mixer=latent, mlp=experts)])


DESIGNS = {"zivitar": zivitar_config, "ramolix": ramolix_config, "mugedra": mugedra_config, "buludra": buludra_config,
           "forisun": forisun_config, "mibezen": mibezen_config}
# what a design is measured beside: the Llama decoder, or the design whose kernels are most like its own
BESIDE = {"zivitar": ("llama",), "ramolix": ("llama",), "mugedra": ("ramolix", "llama"), "buludra": ("mugedra", "llama"),
          "forisun": ("ramolix", "buludra", "llama"), "mibezen": ("forisun", "mugedra", "llama")}


def run_design(which, design="zivitar"):
    """A design (Zivitar, Ramolix, Mugedra, Buludra, Forisun or Mibezen) beside the Llama decoder, Mugedra also beside Ramolix, whose
    mixers (a recurrence behind a short convolution, attention over part of the keys) are most like its own, and
    Buludra also beside Mugedra (two mixers side by side, a recurrence with a matrix state, experts), and Forisun also
    beside Ramolix (latent attention, norms on the sublayers' outputs) and Buludra (experts weighted on their outputs),
    and Mibezen beside Forisun (latent attention, experts) and Mugedra (attention in chunks, experts), at
    equal layer sizes (random weights, four layer runs):
    prompt steps and decode steps timed on the device, and each step's kernels one by one (`Model.profile`).  One
    JSON line per (size, model)."""
    import torch

    import janus_b200
    from janus_b200.engine.step import StepEntry
    for name in which.split(","):
        size = DESIGN_SIZES[name]
        for label in (design,) + BESIDE[design]:
            cfg = llama_like(**size) if label == "llama" else DESIGNS[label](**size)
            model = janus_b200.load_random(cfg, seed=5, dtype="bfloat16", max_tokens=8 * 2176 + 8192 + 1024, max_slots=16,
                                           max_seq_len=16384, norm_std=0.0)
            V = size["vocab"]
            g = torch.Generator().manual_seed(1)

            def toks(n):
                return torch.randint(0, V, (n,), generator=g).tolist()

            def timed(fn, reps):
                for _ in range(3):
                    fn()
                torch.cuda.synchronize()
                a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                a.record()
                for _ in range(reps):
                    fn()
                b.record()
                torch.cuda.synchronize()
                return a.elapsed_time(b) / reps

            out = {"impl": "janus_b200", "design": label, "size": name, "layers": 4, "dtype": "bf16",
                   "data": "synthetic token ids, random-init weights (seed 5)", "config": size}
            for n in (2048, 8192):
                prompt = toks(n)

                def prefill():
                    s = model.alloc_slot()
                    model.step([StepEntry(s, prompt, (n - 1,))])
                    model.free_slot(s)
                ms = timed(prefill, 4)
                out[f"prefill_{n}_ms"] = round(ms, 3)
                out[f"prefill_{n}_tokens_per_s"] = round(n / ms * 1e3, 0)
            slots = [model.alloc_slot() for _ in range(8)]
            model.step([StepEntry(s, toks(2048), ()) for s in slots])
            tok = toks(8)

            def decode():
                model.step([StepEntry(s, (t,), (0,)) for s, t in zip(slots, tok)])
            ms = timed(decode, 32)
            out["decode_batch8_ctx2048_ms"] = round(ms, 4)
            out["decode_batch8_ctx2048_tokens_per_s"] = round(8 / ms * 1e3, 0)
            for s in slots:
                model.free_slot(s)
            prof = model.profile([toks(2048)])
            out["prefill_2048_kernels"] = {k["name"]: [k["launches"], k["ms"]] for k in prof["prefill"]["kernels"]}
            prof = model.profile([toks(2048) for _ in range(8)])
            out["decode_batch8_kernels"] = {k["name"]: [k["launches"], k["ms"]] for k in prof["decode"]["kernels"]}
            model.check()
            print(json.dumps(out), flush=True)
            del model
            torch.cuda.empty_cache()


def run_plan_check():
    """The pick of `ops.gemm_plan` against every alternative it ranks (single-CTA kernel and CTA pairs, K in
    1 to 8 slices) for adding products of three layer sizes at decode and prompt token counts: each variant
    is captured 12 times into a CUDA graph over 4 copies of the weight and timed.  One line per shape with the
    pick, the best alternative and how far the pick is off."""
    import torch

    from janus_b200.kernels import ops
    dev = "cuda:0"

    def timed(fn, reps=12):
        for _ in range(2):
            fn()
        torch.cuda.synchronize()
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g):
            for _ in range(reps):
                fn()
        g.replay()
        torch.cuda.synchronize()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        for _ in range(3):
            g.replay()
        b.record()
        torch.cuda.synchronize()
        return a.elapsed_time(b) / (3 * reps) * 1e3

    shapes = [("1B o", 2048, 2048), ("1B down", 2048, 8192), ("8B o", 4096, 4096), ("8B down", 4096, 14336),
              ("13B o", 5120, 5120), ("13B down", 5120, 13824)]
    for name, N, K in shapes:
        ws = [ops.pack_weight((torch.randn(N, K, device=dev) * 0.02).to(torch.bfloat16)) for _ in range(4)]
        for T in (8, 64, 256, 1024, 2048):
            x = torch.randn(T, K, device=dev).to(torch.bfloat16)
            y = torch.zeros(T, N, device=dev, dtype=torch.float32)
            pick3 = ops.gemm_plan_whole(T, N, K, "add")
            pick = pick3[:2]
            times = {}
            k_tiles = (K + 63) // 64
            for pair in ((False, True) if T >= ops.GEMM_PAIR_MIN_TOKENS else (False,)):
                for split in sorted({1, 2, 3, 4, 6, 8, pick[1]}):
                    if split > 1 and split > max(1, k_tiles // 4):
                        continue
                    if pair and split > 6:
                        continue
                    turn = [0]

                    def fn():
                        turn[0] += 1
                        ops.gemm_bf16(x, ws[turn[0] % 4], y, mode="add", split_k=split, pair=pair)

                    times[(pair, split)] = timed(fn)
            if pick3[2]:      # only the last wave's tiles are cut: a variant of its own
                turn = [0]

                def fn():
                    turn[0] += 1
                    ops.gemm_bf16(x, ws[turn[0] % 4], y, mode="add", split_k=pick3[1], pair=True, whole_tiles=pick3[2])

                pick_us = timed(fn)
            else:
                pick_us = times[pick]
            best = min(times, key=times.get)
            print(json.dumps({"product": name, "tokens": T,
                              "pick": {"pairs": pick[0], "splits": pick[1], "whole_tiles": pick3[2]},
                              "pick_us": round(pick_us, 1), "best": {"pairs": best[0], "splits": best[1]},
                              "best_us": round(times[best], 1),
                              "pick_off_by": round(pick_us / times[best] - 1.0, 4)}), flush=True)
    ops.check_kernel_status(torch.device(dev))


def run_cpu_baseline():
    """The plain implementation (tests/plain_llama.py: whole sequences, no cache, float32 on the host cores)
    timed on the workloads of the two tiny configurations and on one 8B-sized layer.  The reference cannot be
    built or run here; this is the one stand-in that runs, and what it shows is the cost of having no cache
    and no GPU, not the reference's speed."""
    import torch

    sys.path.insert(0, os.path.join(ROOT, "tests"))
    import plain_llama as P
    from helpers import TINY_A, TINY_B, random_tokens

    from janus_b200.config import resolve_architecture
    from janus_b200.weights import RandomCheckpoint

    def weights(cfg, seed):
        arch = resolve_architecture(cfg)
        ck = RandomCheckpoint(arch.weight_specs(arch.config_class.from_dict(cfg)), seed, dtype="float32")
        return {n: ck.tensor(n) for n in ck.names()}

    threads = torch.get_num_threads()
    for name, cfg, seed, lens, new in (("Tiny A", TINY_A, 0, (5, 11, 17), 8), ("Tiny B", TINY_B, 1, (1, 7, 33, 64), 16)):
        w = weights(cfg, seed)
        prompts = [random_tokens(n, cfg["vocab_size"], n) for n in lens]
        P.generate(cfg, w, prompts[0], 2, temperature=0.0)          # warm-up
        t0 = time.perf_counter()
        made = sum(len(P.generate(cfg, w, p, new, temperature=0.0)) for p in prompts)
        dt = time.perf_counter() - t0
        print(json.dumps({"impl": "plain implementation on the host", "workload": name, "prompts": list(lens),
                          "new_tokens_each": new, "value": round(made / dt, 1), "unit": "tokens/s",
                          "wall_s": round(dt, 3), "threads": threads, "dtype": "float32"}), flush=True)
    layer = dict(CONFIG_8B, num_hidden_layers=1, vocab_size=2048, max_position_embeddings=1024)
    w = weights(layer, 2)
    ids = random_tokens(64, 2048, 1)
    P.forward(layer, w, ids)
    t0 = time.perf_counter()
    for _ in range(3):
        P.forward(layer, w, ids)
    dt = (time.perf_counter() - t0) / 3
    flops = 2 * 64 * layer_weight_elems(layer)
    print(json.dumps({"impl": "plain implementation on the host", "workload": "one 8B-sized layer, 64 tokens, whole",
                      "value": round(64 / dt, 1), "unit": "tokens/s", "ms": round(dt * 1e3, 2),
                      "GFLOPs": round(flops / dt / 1e9, 1), "threads": threads, "dtype": "float32"}), flush=True)


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--batch", type=int, default=8, help="batch size of the headline number")
    ap.add_argument("--layers", type=int, default=0, help="fewer layers than the configuration (named in `config`)")
    ap.add_argument("--quick", action="store_true", help="headline batch only")
    ap.add_argument("--no-check", action="store_true",
                    help="skip the comparison with the 32-bit engine before timing (`checked` is then null)")
    ap.add_argument("--deterministic", action="store_true",
                    help="time the headline with the slices of a cut K summed in their fixed order (same bits "
                         "run to run; as JANUS_DETERMINISTIC=1)")
    ap.add_argument("--workload", default="8b", choices=["8b", "1b", "13b"],
                    help="8b: the headline benchmark; 1b / 13b: the other workloads of BASELINE.json, end to end")
    ap.add_argument("--prompt-lengths", nargs="?", const=PROMPT_STEPS, default=None, metavar="SEQSxTOKENS,...",
                    help="time prompt steps at the 8B layer sizes, by default of 96 to 4,096 tokens (one JSON line "
                         "each; --layers, default 8)")
    ap.add_argument("--kernels", action="store_true",
                    help="time the step's hot kernels alone at the 8B layer shapes (one JSON line each)")
    ap.add_argument("--contexts", default=None, metavar="KEYS,...",
                    help="with --kernels: decode attention alone at these context lengths (1 and 8 sequences)")
    ap.add_argument("--head-sizes", default=None, metavar="DIMS,...",
                    help="with --kernels: prompt attention alone at these head sizes, on each kernel that takes them")
    ap.add_argument("--kernel-shape", default="8b", choices=sorted(KERNEL_SHAPES),
                    help="with --kernels: the layer sizes (default: the 8B shape)")
    ap.add_argument("--float32", action="store_true",
                    help="time the true 32-bit path at the 8B layer sizes through generate (one JSON line; --layers, "
                         "default 32)")
    ap.add_argument("--plan-check", action="store_true",
                    help="time the kernel and K-split that `ops.gemm_plan` picks against its alternatives for the "
                         "products of 1B-, 8B- and 13B-sized layers (one JSON line each)")
    ap.add_argument("--cpu-baseline", action="store_true",
                    help="time the plain implementation of tests/ on the host (the only runnable stand-in for the "
                         "reference on this box): Tiny A, Tiny B and one 8B-sized layer (one JSON line each)")
    ap.add_argument("--design", nargs="?", const="2k,4k", default=None, metavar="SIZE,...",
                    help="a second design beside the Llama decoder at equal layer sizes (" + ", ".join(DESIGN_SIZES) +
                         "): prompt and decode throughput and each step's kernels, one JSON line per size and model")
    ap.add_argument("--design-model", choices=sorted(DESIGNS), default="zivitar",
                    help="which design --design measures (default: zivitar)")
    args = ap.parse_args()
    if args.cpu_baseline:
        run_cpu_baseline()
        return 0
    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable":
                          "DaCodeChick/Janus is a Rust workspace that runs WGSL shaders through wgpu (a graphics "
                          "API): pip cannot install it, no cargo/rustc here, no graphics stack on this box"}))
        return 0
    if args.gpus != 1:
        print(f"janus_b200 is a single-GPU library: --gpus {args.gpus} is not supported (run with --gpus 1)")
        return 2
    if args.warmup < 3:
        args.warmup = 3
    if args.kernels:
        run_kernels([int(c) for c in args.contexts.split(",")] if args.contexts else None, args.kernel_shape,
                    [int(c) for c in args.head_sizes.split(",")] if args.head_sizes else None)
        return 0
    if args.float32:
        run_float32(args.layers or 32)
        return 0
    if args.plan_check:
        run_plan_check()
        return 0
    if args.design:
        run_design(args.design, args.design_model)
        return 0
    if args.prompt_lengths:
        run_prompt_lengths(args.layers or 8, args.prompt_lengths)
        return 0
    if args.workload != "8b":
        run_workload(args.workload)
        return 0
    return run_ours(args)


if __name__ == "__main__":
    sys.exit(main())
