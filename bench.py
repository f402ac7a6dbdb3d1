"""Benchmark of the headline metric: decoded tokens per second of a Falcon-7B-shaped model in
bfloat16 with random weights on one B200, batch 8 at context 2,048; plus prefill of 2,048
tokens, decode at batch 1 and 64, the HBM roofline of the decode step, and the same decode rate
end to end through ``generate`` (host tokens in and out).

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--layers L] [--impl ours|reference]

One JSON line on stdout. A "step" is one decode step of the whole batch. Timing: CUDA events on
the launching stream around exactly K steps after W warm-up steps, a synchronize on both sides;
every step reads all weights (13.8 GB, far beyond the 126 MB L2), so no cache flush is needed
between steps. SM clocks and throttle reasons are sampled with nvidia-smi during the timed
region. ``--impl reference`` runs the reference's own FalconForCausalLM.generate from
baseline/_ref on the same shapes.
"""
from __future__ import annotations

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

FALCON_7B = dict(vocab_size=65024, hidden_size=4544, num_hidden_layers=32, num_attention_heads=71,
                 multi_query=True, parallel_attn=True, new_decoder_architecture=False, bias=False, alibi=False,
                 rope_theta=10000.0, layer_norm_epsilon=1e-5, max_position_embeddings=2048,
                 tie_word_embeddings=True, activation="gelu")
# the other two shapes that the reference's Falcon family has (for `--only decode --shape ...`)
FALCON_11B = dict(vocab_size=65024, hidden_size=4096, num_hidden_layers=60, num_attention_heads=32, num_kv_heads=8,
                  new_decoder_architecture=True, num_ln_in_parallel_attn=1, ffn_hidden_size=16384,
                  rope_theta=500042.0, bias=False, alibi=False, layer_norm_epsilon=1e-5,
                  max_position_embeddings=8192, tie_word_embeddings=True, activation="gelu")
FALCON_40B = dict(vocab_size=65024, hidden_size=8192, num_hidden_layers=60, num_attention_heads=128, num_kv_heads=8,
                  new_decoder_architecture=True, ffn_hidden_size=32768, rope_theta=10000.0, bias=False, alibi=False,
                  layer_norm_epsilon=1e-5, max_position_embeddings=2048, tie_word_embeddings=False,
                  activation="gelu")
SHAPES = {"7b": FALCON_7B, "11b": FALCON_11B, "40b": FALCON_40B}
CONTEXT = 2048
PREFILL_TOKENS = 2048
SETTLE_STEPS = 40     # untimed decode steps after a prefill, before the warm-up steps (see run_ours)
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0}


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.isfile(path):
        try:
            raw = json.load(open(path))
            return {"hbm_gbs": float(raw["hbm_gbs"]), "bf16_tflops": float(raw["bf16_tflops"]),
                    "bf16_tflops_sustained": float(raw.get("bf16_tflops_sustained") or raw["bf16_tflops"]),
                    "source": "measured"}
        except Exception:
            pass
    return dict(FALLBACK_PEAKS, source="fallback")


class ClockSampler:
    """nvidia-smi samples of SM clock and throttle reasons while a region runs."""
    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, index: int = 0):
        self.index, self.samples, self.proc = index, [], None

    def __enter__(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits",
                                          "-lms", "100", "-i", str(self.index)], stdout=subprocess.PIPE, text=True)
            self.thread = threading.Thread(target=self._read, daemon=True)
            self.thread.start()
        except OSError:
            self.proc = None
        return self

    def _read(self):
        for line in self.proc.stdout:
            self.samples.append([c.strip() for c in line.split(",")])

    def __exit__(self, *exc):
        if self.proc is not None:
            time.sleep(0.15)
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()
            self.thread.join(timeout=2)

    def summary(self):
        mhz, mx, reasons = [], [], set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for s in self.samples:
            try:
                mhz.append(int(s[0]))
                mx.append(int(s[1]))
            except (ValueError, IndexError):
                continue
            for n, v in zip(names, s[2:6]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        if not mhz:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["no samples"]}
        return {"sm_mhz": int(statistics.median(mhz)), "sm_max_mhz": max(mx), "reasons": sorted(reasons)}


def workload_config(layers, batch):
    """What is run, in the same words for both arms: the layer sizes of Falcon-7B, the batch, the context."""
    h, nh, kvh, d, f, v = shape_sizes(FALCON_7B)
    return {"model": "falcon-7b-shape", "layers": layers, "layers_of_config": FALCON_7B["num_hidden_layers"],
            "hidden": h, "heads": nh, "kv_heads": kvh, "head_dim": d, "ffn": f, "vocab": v, "global_batch": batch,
            "seq_len": CONTEXT, "prompt_tokens": CONTEXT, "weights": "random seed 0", "tokens": "uniform seed 0",
            "parallelism": "none", "sampling": "greedy",
            "l2": "inputs larger than L2 (all weights read per step)"}


def shape_sizes(c):
    """(hidden, heads, K/V heads, head size, feed-forward width, vocabulary) of a shape dictionary."""
    h, nh, v = c["hidden_size"], c["num_attention_heads"], c["vocab_size"]
    f = c.get("ffn_hidden_size") or 4 * h
    kvh = c.get("num_kv_heads", 1) if c.get("new_decoder_architecture") else (1 if c.get("multi_query", True) else nh)
    return h, nh, kvh, h // nh, f, v


def falcon_param_count(c, layers):
    """Weights that a step reads: the layers' matrices and norm vectors and the head matrix (tied or not,
    it is read once; of the embedding table a step reads a row per token). Also the count of one layer."""
    h, nh, kvh, d, f, v = shape_sizes(c)
    norms = 2 if (c.get("new_decoder_architecture") and c.get("num_ln_in_parallel_attn", 2) != 1) or \
        not (c.get("new_decoder_architecture") or c.get("parallel_attn", True)) else 1
    per_layer = (nh + 2 * kvh) * d * h + h * h + 2 * f * h + norms * 2 * h
    return layers * per_layer + v * h + 2 * h, per_layer


def decode_bytes(c, layers, batch, context):
    """Bytes a decode step has to read: every weight it uses once and the cached keys and values of the
    live requests, in bfloat16."""
    h, nh, kvh, d, f, v = shape_sizes(c)
    params, _ = falcon_param_count(c, layers)
    kv = batch * context * layers * 2 * kvh * d * 2
    return 2 * params + kv


def prefill_flops(c, layers, tokens):
    h, nh, kvh, d, f, v = shape_sizes(c)
    gemm = 2 * tokens * layers * ((nh + 2 * kvh) * d * h + h * h + 2 * f * h)
    attn = layers * nh * 2 * 2 * d * tokens * (tokens + 1) / 2      # QK^T and PV over the causal half
    head = 2 * v * h
    return gemm + attn + head


class NoCollection:
    """The engine's guard for stream captures (no cyclic garbage collection inside), looked up when used so
    that `bench.py --gpus 2` and `--impl reference` need not import the package."""

    def __enter__(self):
        from pytorch_transformers_b200.engine.model import NoCollection as Guard
        self.guard = Guard()
        return self.guard.__enter__()

    def __exit__(self, *exc):
        return self.guard.__exit__(*exc)


def run_sample(args):
    """Device time of the selection kernel for the ways of sampling, `--batch` rows of the 7B vocabulary,
    20 launches captured in a CUDA graph (no host time); rows of scale 3 are flat, of scale 6 peaked."""
    import torch

    from pytorch_transformers_b200 import kernels

    torch.cuda.set_device(0)
    rows, vocab = args.batch, SHAPES["7b"]["vocab_size"]
    gen = torch.Generator(device="cuda").manual_seed(0)
    base = torch.randn(rows, vocab, device="cuda", generator=gen)
    work = torch.empty_like(base)
    out = torch.empty(rows, dtype=torch.int32, device="cuda")
    streams = torch.arange(rows, dtype=torch.int64, device="cuda")
    counters = torch.zeros(rows, dtype=torch.int64, device="cuda")
    cases = {"greedy": (3.0, dict(do_sample=False)), "temperature": (3.0, dict(do_sample=True, temperature=0.8)),
             "top_k 50": (3.0, dict(do_sample=True, top_k=50)),
             "top_k 50 top_p 0.9": (3.0, dict(do_sample=True, top_k=50, top_p=0.9, temperature=0.7)),
             "top_k 2000": (3.0, dict(do_sample=True, top_k=2000)),
             "top_p 0.9 peaked": (6.0, dict(do_sample=True, top_p=0.9)),
             "top_p 0.9 flat": (3.0, dict(do_sample=True, top_p=0.9)), "min_p 0.05": (3.0, dict(do_sample=True, min_p=0.05))}
    result = {"only": "sample", "rows": rows, "vocab": vocab, "unit": "us per launch"}
    side = torch.cuda.Stream()
    for name, (scale, opt) in cases.items():
        logits = base * scale
        launch = lambda: kernels.sample(logits, work, out, seed=1, streams=streams, counters=counters, **opt)
        with torch.cuda.stream(side):
            for _ in range(3):
                launch()
            graph = torch.cuda.CUDAGraph()
            with NoCollection(), torch.cuda.graph(graph, stream=side):
                for _ in range(20):
                    launch()
            graph.replay()
            t0, t1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            t0.record()
            for _ in range(5):
                graph.replay()
            t1.record()
        torch.cuda.synchronize()
        result[name] = round(t0.elapsed_time(t1) * 10.0, 1)   # ms for 100 launches -> us for one
    print(json.dumps(result))
    return 0


def run_decode_attention(args):
    """Device time of the two decode attention kernels alone (20 launches in a CUDA graph), `--batch`
    sequences of `--context` cached keys with the heads of `--shape`, for blocks a cluster x clusters a
    sequence."""
    import math

    import torch

    import pytorch_transformers_b200 as ptb
    from pytorch_transformers_b200 import kernels as K
    from pytorch_transformers_b200.cache.paged import Cache
    from pytorch_transformers_b200.engine.batch import StepContext
    from pytorch_transformers_b200.parts.base import CacheNeed

    torch.cuda.set_device(0)
    cfg = ptb.FalconConfig.from_dict(SHAPES[args.shape])
    kv, d, qpk, rows, keys = cfg.kv_heads_eff, cfg.head_dim, cfg.q_per_kv, args.batch, args.context
    cache = Cache([(0, CacheNeed("full", kv, d, 0), None)], rows * (keys + 64), torch.bfloat16, "cuda")
    slots = [cache.open() for _ in range(rows)]
    for slot in slots:
        cache.reserve(slot, keys)
        cache.commit(slot, keys)
    k_pool, v_pool, group = cache.entry_storage(0)
    k_pool.normal_()
    v_pool.normal_()
    ctx = StepContext(cache, slots, [[0]] * rows, 1, [[]] * rows)
    fused = torch.randn(rows, kv * (qpk + 2) * d, device="cuda", dtype=torch.bfloat16)
    rope = K.rope_table(ctx.dev["tok_pos"], (1.0 / (10000 ** (torch.arange(0, d, 2).float() / d))).cuda())
    hpk = min(qpk, 128)
    warps, scale, batch = (hpk + 15) // 16, 1 / math.sqrt(d), ctx.batch_c[group]
    key_split = 1 if warps >= 3 else min(4 if d > 64 else 2, K.decode_max_warps(d) // warps)
    result = {"only": "decode-attention", "shape": args.shape, "batch": rows, "context": keys, "unit": "us per launch"}
    side = torch.cuda.Stream()
    for splits, teams in ((1, 1), (2, 1), (4, 1), (8, 1), (8, 2), (8, 4), (8, 8), (4, 8), (1, 32)):
        if splits * teams * 2 > keys // 64 + 1:
            continue
        launches = {"mma": lambda: K.attention_decode(fused, k_pool, v_pool, batch, rope, None, kv, qpk, d, scale, 0, hpk,
                                                      warps, splits, key_split=key_split, n_teams=teams)}
        if K.attention_decode_tc_supports(d, qpk):
            launches["tcgen05"] = lambda: K.attention_decode_tc(fused, k_pool, v_pool, batch, rope, kv, qpk, d, scale,
                                                                splits, n_teams=teams)
        for name, launch in launches.items():
            with torch.cuda.stream(side):
                for _ in range(3):
                    launch()
                graph = torch.cuda.CUDAGraph()
                with NoCollection(), torch.cuda.graph(graph, stream=side):
                    for _ in range(20):
                        launch()
                graph.replay()
                t0, t1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                t0.record()
                for _ in range(5):
                    graph.replay()
                t1.record()
            torch.cuda.synchronize()
            result[f"{name} {splits}x{teams}"] = round(t0.elapsed_time(t1) * 10.0, 1)
    K.check_device_errors("cuda:0")
    print(json.dumps(result))
    return 0


def run_prefill_attention(args):
    """Device time of the prompt attention kernels alone (10 launches in a CUDA graph, median of 5 replays):
    `--batch` prompts of `--prefill-tokens` tokens after `--past` cached ones, heads of `--shape`."""
    import math

    import torch

    import pytorch_transformers_b200 as ptb
    from pytorch_transformers_b200 import kernels as K
    from pytorch_transformers_b200.cache.paged import Cache
    from pytorch_transformers_b200.engine.batch import StepContext
    from pytorch_transformers_b200.parts.attention import AttentionTiles
    from pytorch_transformers_b200.parts.base import CacheNeed

    torch.cuda.set_device(0)
    cfg = ptb.FalconConfig.from_dict(SHAPES[args.shape])
    kv, d, qpk, rows, new, past = cfg.kv_heads_eff, cfg.head_dim, cfg.q_per_kv, args.batch, args.prefill_tokens, args.past
    heads = kv * qpk
    cache = Cache([(0, CacheNeed("full", kv, d, 0), None)], rows * (past + new + 64), torch.bfloat16, "cuda")
    slots = [cache.open() for _ in range(rows)]
    for slot in slots:
        if past:
            cache.reserve(slot, past)
            cache.commit(slot, past)
    ctx = StepContext(cache, slots, [[0] * new] * rows, 1, [[]] * rows, (AttentionTiles(K),))
    k_pool, v_pool, group = cache.entry_storage(0)
    k_pool.normal_()
    v_pool.normal_()
    tiles, batch = ctx.plan(AttentionTiles.plan_key), ctx.batch_c[group]
    q = torch.randn(rows * new, heads, d, device="cuda", dtype=torch.bfloat16)
    scale = 1 / math.sqrt(d)
    flops = 0.0     # causal: token t of a prompt sees past + t + 1 keys, two products of 2 * d flops per key and head
    flops = rows * heads * 4.0 * d * (new * past + new * (new + 1) / 2)
    result = {"only": "prefill-attention", "shape": args.shape, "batch": rows, "tokens": new, "past": past,
              "GFLOP": round(flops / 1e9, 1)}
    launches = {}
    if tiles.facts["mma_tokens"] == K.TC_TILE_TOKENS and K.attention_tc_supports(d):
        launches["tcgen05"] = lambda: K.attention_tc(q, k_pool, v_pool, batch, tiles.dev["mtile_seq"], tiles.dev["mtile_q0"],
                                                     tiles.facts["n_mma_tiles"], kv, scale, None)
    if "tcgen05" in launches and d == 128 and qpk >= 2:
        def single():
            K.attention_tc_pairs(0)
            try:
                return launches["tcgen05"]()
            finally:
                K.attention_tc_pairs(1)
        launches["tcgen05, a head a block"] = single
    if K.attention_mma_supports(d) and tiles.facts["mma_tokens"] > 1:
        tokens = tiles.facts["mma_tokens"]
        hpk = max(1, min(qpk, 128 // tokens))
        launches["mma"] = lambda: K.attention_mma(q, k_pool, v_pool, batch, tiles.dev["mtile_seq"], tiles.dev["mtile_q0"],
                                                  tiles.facts["n_mma_tiles"], None, kv, scale, 0, tokens, hpk, 8, 1)
    side = torch.cuda.Stream()
    for name, launch in launches.items():
        # 10 launches in a CUDA graph: the host's work for a launch is out of the time
        with torch.cuda.stream(side):
            for _ in range(3):
                launch()
            graph = torch.cuda.CUDAGraph()
            with NoCollection(), torch.cuda.graph(graph, stream=side):
                for _ in range(10):
                    launch()
            graph.replay()
            times = []
            for _ in range(5):
                t0, t1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                t0.record()
                graph.replay()
                t1.record()
                t1.synchronize()
                times.append(t0.elapsed_time(t1) * 100.0)    # ms for 10 launches -> us for one
        torch.cuda.synchronize()
        us = sorted(times)[len(times) // 2]
        result[name] = {"us": round(us, 1), "TFLOPs": round(flops / us / 1e6, 1)}
    K.check_device_errors("cuda:0")
    print(json.dumps(result))
    return 0


def run_mma_cadence(args):
    """Clocks per tcgen05.mma (M = 128, K = 16) for several N, issued back to back by one thread a block on
    operands that are already in shared or tensor memory: one block alone, and two blocks on every SM."""
    import torch

    from pytorch_transformers_b200 import kernels as K

    torch.cuda.set_device(0)
    sms = K.sm_count("cuda:0")
    result = {"only": "mma-cadence", "unit": "clocks per instruction", "reps": 4000}
    for name, tmem, blocks in (("smem A, one block", False, 1), ("tmem A, one block", True, 1),
                               ("smem A, two blocks an SM", False, 2 * sms), ("tmem A, two blocks an SM", True, 2 * sms)):
        row = {}
        for n in (16, 32, 64, 128, 256):
            if tmem and n > 128:
                continue
            K.selftest_mma_cadence("cuda:0", n, 50, tmem, blocks)     # warm-up
            row[str(n)] = round(K.selftest_mma_cadence("cuda:0", n, 1000, tmem, blocks), 1)
        result[name] = row
    K.check_device_errors("cuda:0")
    print(json.dumps(result))
    return 0


def prefill_flops_ragged(c, layers, lengths):
    """Flops of one ragged prefill of prompts of the given lengths (logits for each prompt's last token)."""
    h, nh, kvh, d, f, v = shape_sizes(c)
    total = sum(lengths)
    gemm = 2 * total * layers * ((nh + 2 * kvh) * d * h + h * h + 2 * f * h)
    attn = sum(layers * nh * 2 * 2 * d * n * (n + 1) / 2 for n in lengths)
    return gemm + attn + len(lengths) * 2 * v * h


# BASELINE's runs of the two larger shapes: prompts of seeded uniform lengths in one generate() call
BASELINE_RUNS = {"11b": {"prompts": 8, "shortest": 512, "longest": 8192, "steps": 128},
                 "40b": {"prompts": 16, "shortest": 64, "longest": 2048, "steps": 256}}


def run_config(args, model, cfg, layers, pk):
    """`--only config --shape 11b|40b`: the run that BASELINE names for the shape, through generate():
    prompts of unequal lengths in one ragged prefill (fed in steps of at most 16,384 tokens), then one
    token each for the given number of steps. Device time from CUDA events recorded as each step's tokens
    reach the host; bytes of a decode step from the lengths the sequences really have at mid-run."""
    import torch
    run = BASELINE_RUNS[args.shape]
    gen = torch.Generator().manual_seed(0)
    n, steps = run["prompts"], args.decode_steps or run["steps"]
    lengths = torch.randint(run["shortest"], run["longest"] + 1, (n,), generator=gen).tolist()
    prompts = [torch.randint(0, cfg.vocab_size, (length,), generator=gen).tolist() for length in lengths]
    marks = []

    def on_token(r, tok):
        if r == n - 1:
            ev = torch.cuda.Event(enable_timing=True)
            ev.record()
            marks.append((ev, time.perf_counter()))

    def once():
        marks.clear()
        torch.cuda.synchronize()
        start = torch.cuda.Event(enable_timing=True)
        start.record()
        t0 = time.perf_counter()
        model.generate(prompts, max_new_tokens=steps, eos_token_id=None, max_batch_size=n, on_token=on_token)
        torch.cuda.synchronize()
        return start, t0

    once()                      # sizes the cache, captures the graphs of the decode steps
    with ClockSampler() as sampler:
        start, t0 = once()
    prefill_ms = start.elapsed_time(marks[0][0])
    decode_ms = marks[0][0].elapsed_time(marks[-1][0]) / (len(marks) - 1)
    wall_ms = (marks[-1][1] - marks[0][1]) / (len(marks) - 1) * 1e3
    shape = SHAPES[args.shape]
    h, nh, kvh, d, f, v = shape_sizes(shape)
    params, _ = falcon_param_count(shape, layers)
    mid = sum(lengths) + n * (1 + steps / 2)                       # cached tokens at the middle step
    step_bytes = 2 * params + mid * layers * 2 * kvh * d * 2
    flops = prefill_flops_ragged(shape, layers, lengths)
    print(json.dumps({
        "only": "config", "shape": args.shape, "layers": layers, "layers_of_config": shape["num_hidden_layers"],
        "prompts": n, "prompt_lengths": lengths, "prompt_tokens": sum(lengths), "decode_steps": steps,
        "decode": {"tokens_per_s": round(n / decode_ms * 1e3, 1), "ms_per_step": round(decode_ms, 4),
                   "ms_per_step_wall": round(wall_ms, 4), "bytes_per_step": int(step_bytes),
                   "achieved_GBps": round(step_bytes / decode_ms / 1e6, 1),
                   "frac": round(step_bytes / decode_ms / 1e6 / pk["hbm_gbs"], 4)},
        "prefill": {"tokens_per_s": round(sum(lengths) / prefill_ms * 1e3, 1), "ms": round(prefill_ms, 2),
                    "TFLOPs": round(flops / prefill_ms / 1e9, 1),
                    "frac": round(flops / prefill_ms / 1e9 / pk["bf16_tflops"], 4),
                    "frac_sustained": round(flops / prefill_ms / 1e9 / pk["bf16_tflops_sustained"], 4)},
        "peaks": pk["source"], "clocks": sampler.summary()}))
    return 0


def run_linear(args):
    """`--only linear --rows R`: device time of one linear layer of `--shape` at R rows, for the three ways
    the library has of running it: the weight-streaming kernel (up to 32 rows), the library product
    (cuBLAS through torch) and the tcgen05 kernel (up to 128 rows). 20 launches in a CUDA graph go round
    enough copies of the matrix that every launch reads its weights from HBM, not from L2."""
    import torch

    from pytorch_transformers_b200 import kernels as K

    torch.cuda.set_device(0)
    h, nh, kvh, d, f, v = shape_sizes(SHAPES[args.shape])
    rows = args.rows
    shapes = {"qkv": ((nh + 2 * kvh) * d, h), "out": (h, nh * d), "up": (f, h), "down": (h, f), "head": (v, h)}
    x_cache = {}
    result = {"only": "linear", "shape": args.shape, "rows": rows, "unit": "us per launch (GB/s of the matrix)"}
    side = torch.cuda.Stream()
    for name, (n, k) in shapes.items():
        copies = max(2, -(-(300 << 20) // (n * k * 2)))
        ws = [torch.randn(n, k, device="cuda", dtype=torch.bfloat16) * 0.02 for _ in range(copies)]
        x = x_cache.setdefault(k, torch.randn(rows, k, device="cuda", dtype=torch.bfloat16))
        ways = {"library": lambda w: K.matmul_nt(x, w)}
        if K.skinny_linear_takes(rows, k):
            ways["skinny"] = lambda w: K.skinny_linear(x, w)
        if K.tc_linear_takes(rows, k):
            ways["tcgen05"] = lambda w: K.tc_linear(x, w)
        for way, launch in ways.items():
            with torch.cuda.stream(side):
                for i in range(3):
                    launch(ws[i % copies])
                graph = torch.cuda.CUDAGraph()
                with NoCollection(), torch.cuda.graph(graph, stream=side):
                    for i in range(20):
                        launch(ws[i % copies])
                graph.replay()
                t0, t1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                t0.record()
                for _ in range(5):
                    graph.replay()
                t1.record()
            torch.cuda.synchronize()
            us = t0.elapsed_time(t1) * 10.0
            result[f"{name} {way}"] = [round(us, 1), round(n * k * 2 / us / 1e3)]
        del ws
        torch.cuda.empty_cache()
    K.check_device_errors("cuda:0")
    print(json.dumps(result))
    return 0


def run_fill(args):
    """`--only fill`: device time of the random-weights kernel on one matrix of `--shape`'s feed-forward
    (bfloat16 and float32) and of the whole model of `--layers` layers through from_config."""
    import torch

    import pytorch_transformers_b200 as ptb
    from pytorch_transformers_b200 import kernels as K
    from pytorch_transformers_b200.weights import generator

    torch.cuda.set_device(0)
    h, nh, kvh, d, f, v = shape_sizes(SHAPES[args.shape])
    result = {"only": "fill", "shape": args.shape}
    for dtype, name in ((torch.bfloat16, "bf16"), (torch.float32, "f32")):
        out = torch.empty((f, h), dtype=dtype, device="cuda")
        key = generator.tensor_key(0, "w")
        K.fill_normal(out, key, 0.02)
        torch.cuda.synchronize()
        t0, t1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        t0.record()
        for _ in range(5):
            K.fill_normal(out, key, 0.02)
        t1.record()
        torch.cuda.synchronize()
        ms = t0.elapsed_time(t1) / 5
        result[f"matrix {f}x{h} {name}"] = {"ms": round(ms, 3), "Gvalues_per_s": round(f * h / ms / 1e6, 1),
                                            "GBps_written": round(out.numel() * out.element_size() / ms / 1e6, 1)}
    layers = args.layers or SHAPES[args.shape]["num_hidden_layers"]
    cfg = ptb.FalconConfig.from_dict(dict(SHAPES[args.shape], num_hidden_layers=layers))
    torch.cuda.synchronize()
    t = time.perf_counter()
    model = ptb.AutoModelForCausalLM.from_config(cfg, seed=0, dtype="bfloat16", device="cuda:0")
    torch.cuda.synchronize()
    result["model"] = {"layers": layers, "seconds": round(time.perf_counter() - t, 2),
                       "GB": round(model.weight_bytes() / 1e9, 2)}
    print(json.dumps(result))
    return 0


# ---- Pafevik beside Falcon at equal size (`--only pafevik [--size s|m]`) ----
# Sizes that resemble a served model's layers: the width, 16 or 32 heads of 96 plain + 32 rotated query/key
# entries and values of 128, key/value latents of 512, a recurrence 4/3 of the width wide in 16 blocks with 4
# taps, 64 experts of 1,408 of which a token uses 6 (in 4 of 8 groups). Four layers: latent attention,
# two recurrent layers, latent attention on the first layer's cache entry. Falcon beside it has the same
# width, layers, heads (of 128) and a dense feed-forward as wide as the experts a token uses.
PAFEVIK_SIZES = {"s": dict(width=2048, heads=16, q_rank=768), "m": dict(width=4096, heads=32, q_rank=1536)}


def pafevik_config(size):
    z = PAFEVIK_SIZES[size]
    w, heads = z["width"], z["heads"]
    att = {"heads": heads, "dim": 96, "rot_dim": 32, "vdim": 128, "q_rank": z["q_rank"], "kv_rank": 512,
           "rot": {"base": 10000.0, "dims": 32}, "scale": 128 ** -0.5}
    rec = {"width": w * 4 // 3 // 256 * 256, "blocks": 16, "conv": 4}
    mlp = {"kind": "moe", "expert": {"ff": 1408},
           "router": {"experts": 64, "top": 6, "identity": 0, "scale": 1.0, "groups": {"count": 8, "keep": 4}}}
    layers = [{"type": "latent_attention", "mixer": dict(att), "mlp": mlp}, {"type": "rglru", "mixer": rec, "mlp": mlp},
              {"type": "rglru", "mixer": rec, "mlp": mlp},
              {"type": "latent_attention", "mixer": dict(att, kv_from=0), "mlp": mlp}]
    return {"architecture": "Pafevik", "vocab": 32000, "width": w, "norm": {"eps": 1e-6}, "logit_scale": 1.0, "layers": layers}


def falcon_beside(size):
    z = PAFEVIK_SIZES[size]
    return dict(vocab_size=32000, hidden_size=z["width"], num_hidden_layers=4, num_attention_heads=z["heads"],
                num_kv_heads=z["heads"], new_decoder_architecture=True, num_ln_in_parallel_attn=2,
                ffn_hidden_size=6 * 1408 * 3 // 2, rope_theta=10000.0, bias=False, alibi=False, layer_norm_epsilon=1e-5,
                max_position_embeddings=8192, tie_word_embeddings=False, activation="gelu")


class KernelTimes:
    """Times every call of the kernel module's entry points with a pair of CUDA events while it is on."""
    NAMES = ("gather_rows", "norm", "norm_stream", "add_stream", "residual", "bias_act_", "to_float", "matmul_nt",
             "skinny_linear", "linear_f32", "rope_table", "split_rotate_store", "attention_tc", "attention_mma",
             "attention_generic", "attention_decode", "attention_decode_tc", "latent_store", "latent_attention",
             "latent_unfolded_attention",
             "latent_expand", "block_linear", "rglru_conv", "rglru_scan", "rglru_scan_chunks", "route", "routed_experts", "scale_",
             "embed_sum", "post_norm_add", "qk_norm_store", "linear_attention", "norm_gate", "glu_clamp", "softcap_",
             "dyt", "mlstm", "head_norm_gate", "rope_norm_store", "talk_mix", "embed_rows", "gla", "gla_decay_", "glu_act",
             "delta_prepare", "delta_rule", "expert_rows", "post_norm", "post_norm_pair", "post_norm_experts", "norm_add", "token_gate",
             "round_rows")

    def __init__(self, kernels):
        self.k, self.records, self.saved = kernels, [], {}

    def __enter__(self):
        import torch
        for name in self.NAMES:
            fn = getattr(self.k, name, None)
            if fn is None:
                continue
            self.saved[name] = fn

            def timed(*a, _fn=fn, _name=name, **kw):
                b, e = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                b.record()
                out = _fn(*a, **kw)
                e.record()
                self.records.append((_name, b, e))
                return out
            setattr(self.k, name, timed)
        return self

    def __exit__(self, *exc):
        for name, fn in self.saved.items():
            setattr(self.k, name, fn)

    def table(self):
        import torch
        torch.cuda.synchronize()
        out = {}
        for name, b, e in self.records:
            t = out.setdefault(name, [0, 0.0])
            t[0] += 1
            t[1] += b.elapsed_time(e)
        return {n: {"calls": c, "ms": round(ms, 4)} for n, (c, ms) in sorted(out.items(), key=lambda kv: -kv[1][1])}


def measure_prefill_and_decode(model, args, gen, flush):
    """A prompt of ``args.prefill_tokens`` (median of three after two warm-up runs, L2 flushed before each) and steps
    of ``args.batch`` single tokens at ``args.context`` (replayed graphs), each also once with every kernel call
    between a pair of events."""
    import torch

    from pytorch_transformers_b200 import kernels
    tokens, batch, context = args.prefill_tokens, args.batch, args.context
    vocab = model.spec.vocab_size
    prompt = torch.randint(0, vocab, (1, tokens), generator=gen).tolist()
    cache = model.new_cache(max(tokens + 64, batch * ((context + args.steps + args.warmup + 70) // 64 * 64)))

    def prefill_once():
        s = cache.open()
        flush.zero_()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        model.step(cache, [s], prompt, want="last")
        b.record()
        torch.cuda.synchronize()
        cache.close(s)
        return a.elapsed_time(b)

    times = [prefill_once() for _ in range(2 + 3)][2:]
    with KernelTimes(kernels) as kt:
        prefill_once()
    pre_kernels = kt.table()
    pre_ms = statistics.median(times)
    # decode: `batch` sequences of `context` tokens, then single tokens
    slots = [cache.open() for _ in range(batch)]
    chunk = max(1, 8192 // context)
    for i in range(0, batch, chunk):
        ps = torch.randint(0, vocab, (len(slots[i:i + chunk]), context), generator=gen).tolist()
        model.step(cache, slots[i:i + chunk], ps, want="last")
    one = [[1]] * batch
    for _ in range(args.warmup):
        model.step(cache, slots, one, want="last")
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(args.steps):
        model.step(cache, slots, one, want="last")
    b.record()
    torch.cuda.synchronize()
    dec_ms = a.elapsed_time(b) / args.steps
    graphs, model.use_graphs = model.use_graphs, False
    with KernelTimes(kernels) as kt:
        model.step(cache, slots, one, want="last")
    dec_kernels = kt.table()
    model.use_graphs = graphs
    cache.close_all()
    weights = model.weight_bytes()
    out = {"prefill_ms": round(pre_ms, 3), "prefill_tokens_per_s": round(tokens / pre_ms * 1e3, 1),
           "decode_ms_per_step": round(dec_ms, 4), "decode_tokens_per_s": round(batch / dec_ms * 1e3, 1),
           "weight_GB": round(weights / 1e9, 3), "decode_weight_GBps": round(weights / dec_ms / 1e6, 1),
           "prefill_kernels_ms": pre_kernels,
           # launched one by one the decode step is paced by the host: these are upper bounds
           "decode_kernels_ms": dec_kernels}
    del cache
    torch.cuda.empty_cache()
    return out


def run_pafevik(args):
    import torch

    import pytorch_transformers_b200 as ptb
    from pytorch_transformers_b200 import kernels

    torch.cuda.set_device(0)
    pk = peaks()
    gen = torch.Generator().manual_seed(0)
    tokens, batch, context = args.prefill_tokens, args.batch, args.context
    raw = pafevik_config(args.size)
    models = {"pafevik": ptb.AutoModelForCausalLM.from_config(ptb.PafevikConfig.from_dict(raw), seed=0, dtype="bfloat16"),
              "falcon": ptb.AutoModelForCausalLM.from_config(ptb.FalconConfig.from_dict(falcon_beside(args.size)), seed=0,
                                                             dtype="bfloat16")}
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    result = {"only": "pafevik", "size": args.size, "prefill_tokens": tokens, "batch": batch, "context": context,
              "config": {"width": raw["width"], "layers": len(raw["layers"]), "heads": raw["layers"][0]["mixer"]["heads"]}}
    for name, model in models.items():
        result[name] = measure_prefill_and_decode(model, args, gen, flush)
    # the prompt's kernels against their rooflines (algorithmic FLOPs or bytes; a prompt's launches are paced by the
    # device, so the event pairs around them hold). The kernels of a step of single tokens are listed with their
    # device times under profiles/ (launch lists): launched one by one such a step is paced by the host.
    m = raw["layers"][0]["mixer"]
    H, dk, rank = m["heads"], m["kv_rank"] + m["rot_dim"], m["kv_rank"]
    pairs = tokens * 6

    def per_call(table, key):
        return table[key]["ms"] / table[key]["calls"] if key in table else None

    P, F = result["pafevik"], result["falcon"]
    roof = {}
    t = per_call(P["prefill_kernels_ms"], "latent_attention")
    if t:
        roof["latent_attention_prefill_TFLOPs_as_run"] = round(H * tokens * (tokens + 1) / 2 * 2 * (dk + rank) / t / 1e9, 1)
        roof["latent_attention_prefill_frac_of_burst"] = round(roof["latent_attention_prefill_TFLOPs_as_run"] / pk["bf16_tflops"], 3)
    t = per_call(P["prefill_kernels_ms"], "latent_unfolded_attention")
    if t:   # gather, unfolding product, scatter, query layout, the tcgen05 kernel and the gate together
        m0 = raw["layers"][0]["mixer"]
        flops = H * tokens * (tokens + 1) / 2 * 2 * (m0["dim"] + m0["rot_dim"] + m0["vdim"]) + \
            2 * tokens * rank * H * (m0["dim"] + m0["vdim"])
        roof["latent_attention_prefill_unfolded_TFLOPs"] = round(flops / t / 1e9, 1)
        roof["latent_attention_prefill_unfolded_frac_of_burst"] = round(flops / t / 1e9 / pk["bf16_tflops"], 3)
    t = per_call(F["prefill_kernels_ms"], "attention_tc")
    if t:
        roof["falcon_attention_prefill_TFLOPs"] = round(H * tokens * (tokens + 1) / 2 * 4 * 128 / t / 1e9, 1)
        roof["falcon_attention_prefill_frac_of_burst"] = round(roof["falcon_attention_prefill_TFLOPs"] / pk["bf16_tflops"], 3)
    t = per_call(P["prefill_kernels_ms"], "routed_experts")
    if t:
        roof["experts_prefill_TFLOPs"] = round(pairs * 3 * 2 * raw["width"] * 1408 / t / 1e9, 1)
        roof["experts_prefill_frac_of_burst"] = round(roof["experts_prefill_TFLOPs"] / pk["bf16_tflops"], 3)
    ff = falcon_beside(args.size)["ffn_hidden_size"]
    t = F["prefill_kernels_ms"].get("matmul_nt")
    if t:   # all of Falcon's products of the prompt, the library's
        h = raw["width"]
        flops = 4 * 2 * tokens * (3 * h * h + h * h + 2 * ff * h)
        roof["falcon_library_products_TFLOPs"] = round(flops / t["ms"] / 1e9, 1)
        roof["falcon_library_products_frac_of_burst"] = round(roof["falcon_library_products_TFLOPs"] / pk["bf16_tflops"], 3)
    t = per_call(P["prefill_kernels_ms"], "rglru_scan_chunks")
    if t:
        R = raw["layers"][1]["mixer"]["width"]
        roof["rglru_scan_prefill_GBps"] = round(tokens * R * (8 + 2 + 2 + 2) / t / 1e6, 1)     # gates, u, y in; out
        roof["rglru_scan_prefill_frac_of_hbm"] = round(roof["rglru_scan_prefill_GBps"] / pk["hbm_gbs"], 3)
    result["roofline"] = roof
    result["peaks"] = pk
    print(json.dumps(result))
    return 0


# ---- Zalunex beside Pafevik at equal size (`--only zalunex [--size s|m]`) ----
# Sizes that resemble a served model's layers: the width; a pair mixer of 16 or 32 attention heads of 128 on a
# quarter as many K/V heads with a window of 1,024, a sink and a gate, beside as many linear-attention heads of 128
# with decays 1 - 2^-(3 + 5 h / heads); four layers whose feed-forwards take turns: a clamped gated unit 4 x the
# width wide, then 64 plain experts of 1,408 of which a token uses 6. Pafevik beside it is `--only pafevik`'s model
# of the same width, heads, layers and experts: the library's other design with a float32 stream, a per-sequence
# state and routed experts.
def zalunex_config(size):
    z = PAFEVIK_SIZES[size]
    w, heads = z["width"], z["heads"]
    mixer = {"left": {"heads": heads, "kv_heads": heads // 4, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": 1024}},
             "right": {"heads": heads, "dim": 128, "vdim": 128, "decay": [1.0 - 2.0 ** -(3 + 5 * h / heads) for h in range(heads)]},
             "left_scale": 1.0, "right_scale": 1.0}
    glu = {"kind": "dense", "ff": 4 * w, "limit": 7.0}
    moe = {"kind": "moe", "expert": {"ff": 1408}, "router": {"experts": 64, "top": 6}}
    return {"architecture": "Zalunex", "vocab": 32000, "width": w, "max_positions": 16384, "norm": {"eps": 1e-6},
            "residual_mult": 0.5, "logit_softcap": 30.0,
            "layers": [{"type": "parallel", "mixer": mixer, "mlp": m} for m in (glu, moe, glu, moe)]}


def run_zalunex(args):
    import torch

    import pytorch_transformers_b200 as ptb

    torch.cuda.set_device(0)
    pk = peaks()
    gen = torch.Generator().manual_seed(0)
    tokens, batch, context = args.prefill_tokens, args.batch, args.context
    raw = zalunex_config(args.size)
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    result = {"only": "zalunex", "size": args.size, "prefill_tokens": tokens, "batch": batch, "context": context,
              "config": {"width": raw["width"], "layers": len(raw["layers"]), "heads": raw["layers"][0]["mixer"]["left"]["heads"]}}
    for name, make in (("zalunex", lambda: ptb.AutoModelForCausalLM.from_config(ptb.ZalunexConfig.from_dict(raw), seed=0, dtype="bfloat16")),
                       ("pafevik", lambda: ptb.AutoModelForCausalLM.from_config(ptb.PafevikConfig.from_dict(pafevik_config(args.size)),
                                                                               seed=0, dtype="bfloat16"))):
        model = make()
        result[name] = measure_prefill_and_decode(model, args, gen, flush)
        del model
        torch.cuda.empty_cache()
    # kernels of the prompt against their rooflines (algorithmic FLOPs or bytes over the time between the event pair
    # around the call; a prompt's launches are paced by the device)
    Z, P = result["zalunex"], result["pafevik"]
    l, r, w = raw["layers"][0]["mixer"]["left"], raw["layers"][0]["mixer"]["right"], raw["width"]

    def per_call(table, key):
        return table[key]["ms"] / table[key]["calls"] if key in table else None

    roof = {}
    seen = sum(min(t + 1, l["mask"]["size"]) for t in range(tokens))        # (query, key) pairs inside the window
    for key in ("attention_generic", "attention_mma"):
        t = per_call(Z["prefill_kernels_ms"], key)
        if t:
            roof[f"sink_{key}_prefill_TFLOPs"] = round(l["heads"] * seen * 2 * (l["dim"] + l["vdim"]) / t / 1e9, 1)
            roof[f"sink_{key}_prefill_frac_of_burst"] = round(roof[f"sink_{key}_prefill_TFLOPs"] / pk["bf16_tflops"], 4)
    t = per_call(Z["prefill_kernels_ms"], "linear_attention")
    if t:   # per chunk of 64: scores, scores x values, queries x state, keys x values
        flops = r["heads"] * tokens * 2 * (64 * r["dim"] / 2 + 64 * r["vdim"] / 2 + 2 * r["dim"] * r["vdim"])
        roof["linear_attention_prefill_TFLOPs"] = round(flops / t / 1e9, 1)
        roof["linear_attention_prefill_frac_of_burst"] = round(roof["linear_attention_prefill_TFLOPs"] / pk["bf16_tflops"], 4)
        io = tokens * r["heads"] * (2 * (2 * r["dim"] + r["vdim"]) + 4 * r["vdim"])      # q, k, v in; float32 rows out
        roof["linear_attention_prefill_GBps"] = round(io / t / 1e6, 1)
        roof["linear_attention_prefill_frac_of_hbm"] = round(roof["linear_attention_prefill_GBps"] / pk["hbm_gbs"], 4)
    t = per_call(P["prefill_kernels_ms"], "rglru_scan_chunks")
    if t:
        R = pafevik_config(args.size)["layers"][1]["mixer"]["width"]
        roof["pafevik_rglru_scan_prefill_GBps"] = round(tokens * R * (8 + 2 + 2 + 2) / t / 1e6, 1)
        roof["pafevik_rglru_scan_prefill_frac_of_hbm"] = round(roof["pafevik_rglru_scan_prefill_GBps"] / pk["hbm_gbs"], 4)
    pairs = tokens * 6
    t = per_call(Z["prefill_kernels_ms"], "routed_experts")
    if t:
        roof["experts_prefill_TFLOPs"] = round(pairs * 2 * 2 * w * 1408 / t / 1e9, 1)
        roof["experts_prefill_frac_of_burst"] = round(roof["experts_prefill_TFLOPs"] / pk["bf16_tflops"], 4)
    t = per_call(P["prefill_kernels_ms"], "routed_experts")
    if t:
        roof["pafevik_experts_prefill_TFLOPs"] = round(pairs * 3 * 2 * w * 1408 / t / 1e9, 1)
        roof["pafevik_experts_prefill_frac_of_burst"] = round(roof["pafevik_experts_prefill_TFLOPs"] / pk["bf16_tflops"], 4)
    t = Z["prefill_kernels_ms"].get("matmul_nt")
    if t:   # all library products of the prompt: the pairs' two products a layer, the gated units' two
        n_in = (l["heads"] + l["kv_heads"]) * l["dim"] + l["kv_heads"] * l["vdim"] + l["heads"] + 2 * r["heads"] * (r["dim"] + r["vdim"])
        n_out = l["heads"] * l["vdim"] + r["heads"] * r["vdim"]
        flops = 2 * tokens * (4 * w * (n_in + n_out) + 2 * 3 * w * 4 * w)
        roof["library_products_TFLOPs"] = round(flops / t["ms"] / 1e9, 1)
        roof["library_products_frac_of_burst"] = round(roof["library_products_TFLOPs"] / pk["bf16_tflops"], 4)
    for key, bytes_per_row in (("post_norm_add", w * (4 + 4 + 4 + 2)), ("norm_gate", r["heads"] * r["vdim"] * (4 + 2 + 2)),
                               ("glu_clamp", 4 * w * (2 + 2 + 2)), ("qk_norm_store", (l["heads"] + 2 * l["kv_heads"]) * l["dim"] * 4)):
        t = per_call(Z["prefill_kernels_ms"], key)
        if t:
            roof[f"{key}_prefill_GBps"] = round(tokens * bytes_per_row / t / 1e6, 1)
            roof[f"{key}_prefill_frac_of_hbm"] = round(roof[f"{key}_prefill_GBps"] / pk["hbm_gbs"], 4)
    t = per_call(P["prefill_kernels_ms"], "norm_stream")
    if t:
        roof["pafevik_norm_stream_prefill_GBps"] = round(tokens * w * (4 + 2) / t / 1e6, 1)
        roof["pafevik_norm_stream_prefill_frac_of_hbm"] = round(roof["pafevik_norm_stream_prefill_GBps"] / pk["hbm_gbs"], 4)
    result["roofline"] = roof
    result["peaks"] = pk
    print(json.dumps(result))
    return 0


# ---- Pogezen beside Zalunex at equal size (`--only pogezen [--size s|m]`) ----
# Sizes that resemble a served model's layers: the width; four layers that take turns between a matrix memory of 16
# or 32 heads of 128 x 128 with capped exponential gates and an attention of as many heads of 128 on a quarter as many
# K/V heads, rotated on half of each head with a stretched rotation, a window of 1,024 that keeps the first 4 tokens,
# mixed softmax weights and mixed values; an input convolution of 4 taps; squared-relu feed-forwards 4 x the width
# wide. Zalunex beside it is `--only zalunex`'s model of the same width, heads and layers: the library's other design
# with a float32 stream, a windowed attention and a matrix state per head.
def pogezen_config(size):
    z = PAFEVIK_SIZES[size]
    w, heads = z["width"], z["heads"]
    mem = {"heads": heads, "dim": 128, "vdim": 128, "gate_cap": 15.0}
    att = {"heads": heads, "kv_heads": heads // 4, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
           "mask": {"size": 1024, "keep_first": 4},
           "rot": {"base": 10000.0, "dims": 64, "scaling": {"factor": 8.0, "original": 2048, "fast": 32.0, "slow": 1.0}},
           "v_mix": True}
    mlp = {"kind": "dense", "ff": 4 * w}
    return {"architecture": "Pogezen", "vocab": 32000, "width": w, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
            "canon": {"taps": 4},
            "layers": [{"type": t, "mixer": dict(m), "mlp": mlp} for t, m in (("mlstm", mem), ("attention", att)) * 2]}


def run_pogezen(args):
    import torch

    import pytorch_transformers_b200 as ptb

    torch.cuda.set_device(0)
    pk = peaks()
    gen = torch.Generator().manual_seed(0)
    tokens, batch, context = args.prefill_tokens, args.batch, args.context
    raw = pogezen_config(args.size)
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    mem, att, w = raw["layers"][0]["mixer"], raw["layers"][1]["mixer"], raw["width"]
    result = {"only": "pogezen", "size": args.size, "prefill_tokens": tokens, "batch": batch, "context": context,
              "config": {"width": w, "layers": len(raw["layers"]), "heads": att["heads"]}}
    for name, make in (("pogezen", lambda: ptb.AutoModelForCausalLM.from_config(ptb.PogezenConfig.from_dict(raw), seed=0, dtype="bfloat16")),
                       ("zalunex", lambda: ptb.AutoModelForCausalLM.from_config(ptb.ZalunexConfig.from_dict(zalunex_config(args.size)),
                                                                               seed=0, dtype="bfloat16"))):
        model = make()
        result[name] = measure_prefill_and_decode(model, args, gen, flush)
        del model
        torch.cuda.empty_cache()
    G, Z = result["pogezen"], result["zalunex"]

    def per_call(table, key):
        return table[key]["ms"] / table[key]["calls"] if key in table else None

    roof = {}
    H, K, d, vd = att["heads"], att["kv_heads"], att["dim"], att["vdim"]
    keep, size = att["mask"]["keep_first"], att["mask"]["size"]
    seen = sum(min(t + 1, size) + max(0, min(keep, t + 1 - size)) for t in range(tokens))     # visible (query, key) pairs
    # the attention with mixed weights: scores of every head, then every head's weights on every K/V head's values
    for key in ("attention_generic", "attention_mma"):
        t = per_call(G["prefill_kernels_ms"], key)
        if t:
            roof[f"talk_{key}_prefill_TFLOPs_as_run"] = round(H * seen * 2 * (d + K * vd) / t / 1e9, 1)
            roof[f"talk_{key}_prefill_TFLOPs_needed"] = round(H * seen * 2 * (d + vd) / t / 1e9, 1)
            roof[f"talk_{key}_prefill_frac_of_burst"] = round(roof[f"talk_{key}_prefill_TFLOPs_as_run"] / pk["bf16_tflops"], 4)
        t = per_call(Z["prefill_kernels_ms"], key)
        if t:
            zl = zalunex_config(args.size)["layers"][0]["mixer"]["left"]
            zseen = sum(min(t_ + 1, zl["mask"]["size"]) for t_ in range(tokens))
            roof[f"zalunex_{key}_prefill_TFLOPs"] = round(zl["heads"] * zseen * 2 * (zl["dim"] + zl["vdim"]) / t / 1e9, 1)
            roof[f"zalunex_{key}_prefill_frac_of_burst"] = round(roof[f"zalunex_{key}_prefill_TFLOPs"] / pk["bf16_tflops"], 4)
    mh, md, mv = mem["heads"], mem["dim"], mem["vdim"]
    t = per_call(G["prefill_kernels_ms"], "mlstm")
    if t:   # per chunk of 64: scores, scores x values, queries x state, keys x values; q, k, v, gates in, float32 rows out
        flops = mh * tokens * 2 * (64 * md / 2 + 64 * mv / 2 + 2 * md * mv)
        io = tokens * mh * (2 * (2 * md + mv) + 8 + 4 * mv)
        roof["mlstm_prefill_TFLOPs"] = round(flops / t / 1e9, 1)
        roof["mlstm_prefill_GBps"] = round(io / t / 1e6, 1)
        roof["mlstm_prefill_frac_of_hbm"] = round(roof["mlstm_prefill_GBps"] / pk["hbm_gbs"], 4)
    t = per_call(Z["prefill_kernels_ms"], "linear_attention")
    if t:
        r = zalunex_config(args.size)["layers"][0]["mixer"]["right"]
        io = tokens * r["heads"] * (2 * (2 * r["dim"] + r["vdim"]) + 4 * r["vdim"])
        roof["zalunex_linear_attention_prefill_GBps"] = round(io / t / 1e6, 1)
        roof["zalunex_linear_attention_prefill_frac_of_hbm"] = round(roof["zalunex_linear_attention_prefill_GBps"] / pk["hbm_gbs"], 4)
    t = G["prefill_kernels_ms"].get("matmul_nt")
    if t:   # all library products of the prompt
        n_mem = 2 * mh * md + 2 * mh * mv + 2 * mh + mh * mv
        n_att = (H + K) * d + K * vd + H * vd
        flops = 2 * tokens * w * (2 * n_mem + 2 * n_att + 4 * 2 * 4 * w)
        roof["library_products_TFLOPs"] = round(flops / t["ms"] / 1e9, 1)
        roof["library_products_frac_of_burst"] = round(roof["library_products_TFLOPs"] / pk["bf16_tflops"], 4)
    # the norm kernels of a prompt: the first reads the stream and writes normed rows (4 + 2 bytes a column), the others
    # also read the float32 sums still to be added and write the new stream (4 + 4 + 4 + 2); the last norms one row
    norms = sum(2 if layer["mlp"] is not None else 1 for layer in raw["layers"])
    dyt_calls = G["prefill_kernels_ms"].get("dyt", {}).get("calls", norms + 1)
    dyt_row = w * ((4 + 2) + (norms - 1) * (4 + 4 + 4 + 2)) / dyt_calls
    for key, bytes_per_row in (("dyt", dyt_row), ("head_norm_gate", mh * mv * (4 + 2 + 2)),
                               ("rope_norm_store", ((H + K) * d + K * vd) * 4), ("talk_mix", H * vd * (4 * K + 2)),
                               ("mlstm_gates", 0)):
        t = per_call(G["prefill_kernels_ms"], key)
        if t and bytes_per_row:
            roof[f"{key}_prefill_GBps"] = round(tokens * bytes_per_row / t / 1e6, 1)
            roof[f"{key}_prefill_frac_of_hbm"] = round(roof[f"{key}_prefill_GBps"] / pk["hbm_gbs"], 4)
    zw = zalunex_config(args.size)["width"]
    for key, bytes_per_row in (("post_norm_add", zw * (4 + 4 + 4 + 2)), ("norm_gate", H * 128 * (4 + 2 + 2)),
                               ("qk_norm_store", (H + 2 * K) * 128 * 4)):
        t = per_call(Z["prefill_kernels_ms"], key)
        if t:
            roof[f"zalunex_{key}_prefill_GBps"] = round(tokens * bytes_per_row / t / 1e6, 1)
            roof[f"zalunex_{key}_prefill_frac_of_hbm"] = round(roof[f"zalunex_{key}_prefill_GBps"] / pk["hbm_gbs"], 4)
    result["roofline"] = roof
    result["peaks"] = pk
    print(json.dumps(result))
    return 0

# ---- Figudra beside Zalunex at equal size (`--only figudra [--size s|m]`) ----
# Sizes that resemble a served model's layers: the width; four parallel layers: an attention of 16 or 32 heads of 128 on a
# quarter as many K/V heads with normed and partly rotated queries and keys, a window of 1,024 that keeps the first 4
# tokens and one added to the softmax's denominator, over a gated GELU unit 4 x the width wide; a gated linear attention
# of as many heads of 128 x 128 whose decays come through a rank of 64, over 64 experts of 1,408 of which a token uses 6
# (in 4 of 8 groups) and a shared expert of 2,816; a full attention with a query temperature, capped scores and a gate
# per entry over the same experts; a gated linear attention over the gated unit. Zalunex beside it is `--only zalunex`'s
# model of the same width, heads, layers and experts: the library's other design with a float32 stream, a windowed
# attention with a sink and a gate, a linear attention with a state per head and routed experts.
def figudra_config(size):
    z = PAFEVIK_SIZES[size]
    w, heads = z["width"], z["heads"]
    win = {"heads": heads, "kv_heads": heads // 4, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
           "mask": {"size": 1024, "keep_first": 4}, "rot": {"base": 10000.0, "dims": 64, "scaling": {"factor": 8.0}}}
    full = {"heads": heads, "kv_heads": heads // 4, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 30.0,
            "q_temp": {"coef": 0.5, "every": 512}}
    lin = {"heads": heads, "dim": 128, "vdim": 128, "tau": 16.0, "rank": 64}
    glu = {"kind": "dense", "ff": 4 * w}
    moe = {"kind": "moe", "expert": {"ff": 1408}, "shared": {"ff": 2816},
           "router": {"experts": 64, "top": 6, "scale": 2.0, "groups": {"count": 8, "keep": 4}}}
    return {"architecture": "Figudra", "vocab": 32000, "width": w, "norm": {"eps": 1e-6},
            "layers": [{"type": t, "mixer": dict(m), "mlp": f} for t, m, f in
                       (("attention_2", win, glu), ("gla", lin, moe), ("attention", full, moe), ("gla", lin, glu))]}


def run_figudra(args):
    import torch

    import pytorch_transformers_b200 as ptb

    torch.cuda.set_device(0)
    pk = peaks()
    gen = torch.Generator().manual_seed(0)
    tokens, batch, context = args.prefill_tokens, args.batch, args.context
    raw = figudra_config(args.size)
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    win, lin, w = raw["layers"][0]["mixer"], raw["layers"][1]["mixer"], raw["width"]
    result = {"only": "figudra", "size": args.size, "prefill_tokens": tokens, "batch": batch, "context": context,
              "config": {"width": w, "layers": len(raw["layers"]), "heads": win["heads"]}}
    for name, make in (("figudra", lambda: ptb.AutoModelForCausalLM.from_config(ptb.FigudraConfig.from_dict(raw), seed=0, dtype="bfloat16")),
                       ("zalunex", lambda: ptb.AutoModelForCausalLM.from_config(ptb.ZalunexConfig.from_dict(zalunex_config(args.size)),
                                                                               seed=0, dtype="bfloat16"))):
        model = make()
        result[name] = measure_prefill_and_decode(model, args, gen, flush)
        del model
        torch.cuda.empty_cache()
    F, Z = result["figudra"], result["zalunex"]

    def per_call(table, key):
        return table[key]["ms"] / table[key]["calls"] if key in table else None

    roof = {}
    H, G, d, vd = win["heads"], win["kv_heads"], win["dim"], win["vdim"]
    keep, size = win["mask"]["keep_first"], win["mask"]["size"]
    seen = sum(min(t + 1, size) + max(0, min(keep, t + 1 - size)) for t in range(tokens))     # pairs the windowed layer sees
    full = tokens * (tokens + 1) // 2                                                         # pairs the full layer sees
    zl, zr = zalunex_config(args.size)["layers"][0]["mixer"]["left"], zalunex_config(args.size)["layers"][0]["mixer"]["right"]
    zseen = sum(min(t_ + 1, zl["mask"]["size"]) for t_ in range(tokens))
    for key in ("attention_generic", "attention_mma"):
        t = F["prefill_kernels_ms"].get(key)
        if t:   # one windowed layer and one full layer share the kernel and the table's row
            roof[f"{key}_prefill_TFLOPs"] = round(H * (seen + full) * 2 * (d + vd) / t["ms"] / 1e9, 1)
            roof[f"{key}_prefill_frac_of_burst"] = round(roof[f"{key}_prefill_TFLOPs"] / pk["bf16_tflops"], 4)
        t = per_call(Z["prefill_kernels_ms"], key)
        if t:
            roof[f"zalunex_{key}_prefill_TFLOPs"] = round(zl["heads"] * zseen * 2 * (zl["dim"] + zl["vdim"]) / t / 1e9, 1)
            roof[f"zalunex_{key}_prefill_frac_of_burst"] = round(roof[f"zalunex_{key}_prefill_TFLOPs"] / pk["bf16_tflops"], 4)
    lh, ld, lv = lin["heads"], lin["dim"], lin["vdim"]
    t = per_call(F["prefill_kernels_ms"], "gla")
    if t:   # q, k, v and the decays' logarithms in, float32 rows out; per token and head: own sum, outputs, state
        io = tokens * lh * (2 * (2 * ld + lv) + 4 * ld + 4 * lv)
        roof["gla_prefill_GBps"] = round(io / t / 1e6, 1)
        roof["gla_prefill_frac_of_hbm"] = round(roof["gla_prefill_GBps"] / pk["hbm_gbs"], 4)
        roof["gla_prefill_TFLOPs_fp32"] = round(lh * tokens * 2 * 3 * ld * lv / t / 1e9, 1)
    t = per_call(Z["prefill_kernels_ms"], "linear_attention")
    if t:
        io = tokens * zr["heads"] * (2 * (2 * zr["dim"] + zr["vdim"]) + 4 * zr["vdim"])
        roof["zalunex_linear_attention_prefill_GBps"] = round(io / t / 1e6, 1)
        roof["zalunex_linear_attention_prefill_frac_of_hbm"] = round(roof["zalunex_linear_attention_prefill_GBps"] / pk["hbm_gbs"], 4)
    pairs = tokens * 6
    t = per_call(F["prefill_kernels_ms"], "routed_experts")
    if t:
        roof["experts_prefill_TFLOPs"] = round(pairs * 3 * 2 * w * 1408 / t / 1e9, 1)
        roof["experts_prefill_frac_of_burst"] = round(roof["experts_prefill_TFLOPs"] / pk["bf16_tflops"], 4)
    t = per_call(Z["prefill_kernels_ms"], "routed_experts")
    if t:
        roof["zalunex_experts_prefill_TFLOPs"] = round(pairs * 2 * 2 * w * 1408 / t / 1e9, 1)
        roof["zalunex_experts_prefill_frac_of_burst"] = round(roof["zalunex_experts_prefill_TFLOPs"] / pk["bf16_tflops"], 4)
    t = F["prefill_kernels_ms"].get("matmul_nt")
    if t:   # all library products of the prompt: projections in and out of the four mixers, the decays' two, gated units, shared experts, head
        n_att = 2 * ((H + G) * d + G * vd + H * vd) + H * vd
        n_lin = 2 * (2 * lh * ld + 3 * lh * lv)
        flops = 2 * tokens * (w * (n_att + n_lin) + 2 * (64 * w + 64 * lh * ld) + 2 * 3 * w * 4 * w + 2 * 3 * w * 2816)
        roof["library_products_TFLOPs"] = round(flops / t["ms"] / 1e9, 1)
        roof["library_products_frac_of_burst"] = round(roof["library_products_TFLOPs"] / pk["bf16_tflops"], 4)
    for key, bytes_per_row in (("norm_stream", w * (4 + 4 + 4 + 2)), ("head_norm_gate", lh * lv * (4 + 2 + 2)),
                               ("rope_norm_store", ((H + G) * d + G * vd) * 4), ("gla_decay_", lh * ld * 8)):
        t = per_call(F["prefill_kernels_ms"], key)
        if t:
            roof[f"{key}_prefill_GBps"] = round(tokens * bytes_per_row / t / 1e6, 1)
            roof[f"{key}_prefill_frac_of_hbm"] = round(roof[f"{key}_prefill_GBps"] / pk["hbm_gbs"], 4)
    t = F["prefill_kernels_ms"].get("glu_act")
    if t:   # two gated units of 4 w and two shared experts of 2,816 columns: gate and up in, product out
        roof["glu_act_prefill_GBps"] = round(tokens * 6 * (2 * 4 * w + 2 * 2816) / t["ms"] / 1e6, 1)
        roof["glu_act_prefill_frac_of_hbm"] = round(roof["glu_act_prefill_GBps"] / pk["hbm_gbs"], 4)
    zw = zalunex_config(args.size)["width"]
    for key, bytes_per_row in (("post_norm_add", zw * (4 + 4 + 4 + 2)), ("norm_gate", zr["heads"] * zr["vdim"] * (4 + 2 + 2)),
                               ("qk_norm_store", (zl["heads"] + 2 * zl["kv_heads"]) * 128 * 4), ("glu_clamp", 4 * zw * 6)):
        t = per_call(Z["prefill_kernels_ms"], key)
        if t:
            roof[f"zalunex_{key}_prefill_GBps"] = round(tokens * bytes_per_row / t / 1e6, 1)
            roof[f"zalunex_{key}_prefill_frac_of_hbm"] = round(roof[f"zalunex_{key}_prefill_GBps"] / pk["hbm_gbs"], 4)
    result["roofline"] = roof
    result["peaks"] = pk
    print(json.dumps(result))
    return 0


# ---- Vesidra beside Pafevik at equal size (`--only vesidra [--size s|m]`) ----
# Sizes that resemble a served model's layers: the width; four parallel layers of latent attention with 16 or 32 heads of
# 96 plain + 32 rotated query/key entries (YaRN frequencies) and values of 128, a key/value latent of 512 and a gate per
# head; layers 0 and 2 over a gated unit 4 x the width wide, layers 1 and 3 over 64 plain experts of 1,408 of which a token
# uses 6 and a shared expert of 2,816. Pafevik beside it has four layers of latent attention of the same heads, sizes and
# latent (queries through a latent of their own, a gate per entry) over 64 gated experts of 1,408 of which a token uses 6.
# `vesidra_192` is Vesidra with heads of 128 plain + 64 rotated entries.
def vesidra_config(size, dim=96, rot_dim=32):
    z = PAFEVIK_SIZES[size]
    w, heads = z["width"], z["heads"]
    att = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": 128, "kv_rank": 512, "scale": (dim + rot_dim) ** -0.5,
           "rot": {"base": 10000.0, "dims": rot_dim, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    glu = {"kind": "dense", "ff": 4 * w}
    moe = {"kind": "moe", "expert": {"ff": 1408}, "shared": {"ff": 2816}, "router": {"experts": 64, "top": 6}}
    return {"architecture": "Vesidra", "vocab": 32000, "width": w, "embedding": {"scale": w ** 0.5}, "norm": {"eps": 1e-6},
            "layers": [{"type": "latent_attention", "mixer": dict(att), "mlp": f} for f in (glu, moe, glu, moe)]}


def pafevik_attention_config(size):
    raw = pafevik_config(size)
    raw["layers"] = [dict(raw["layers"][0], mixer=dict(raw["layers"][0]["mixer"])) for _ in range(4)]
    return raw


def run_vesidra(args):
    import torch

    import pytorch_transformers_b200 as ptb

    torch.cuda.set_device(0)
    pk = peaks()
    gen = torch.Generator().manual_seed(0)
    tokens, batch, context = args.prefill_tokens, args.batch, args.context
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    raws = {"vesidra": vesidra_config(args.size), "vesidra_192": vesidra_config(args.size, 128, 64),
            "pafevik": pafevik_attention_config(args.size)}
    w = raws["vesidra"]["width"]
    result = {"only": "vesidra", "size": args.size, "prefill_tokens": tokens, "batch": batch, "context": context,
              "config": {"width": w, "layers": 4, "heads": raws["vesidra"]["layers"][0]["mixer"]["heads"]}}
    for name, raw in raws.items():
        cls = ptb.PafevikConfig if name == "pafevik" else ptb.VesidraConfig
        model = ptb.AutoModelForCausalLM.from_config(cls.from_dict(raw), seed=0, dtype="bfloat16")
        result[name] = measure_prefill_and_decode(model, args, gen, flush)
        del model
        torch.cuda.empty_cache()

    roof = {}
    pairs, scored = tokens * 6, tokens * (tokens + 1) // 2

    def put(name, value, peak, unit):
        roof[f"{name}_{unit}"] = round(value, 1)
        roof[f"{name}_frac_of_{'hbm' if unit == 'GBps' else 'burst'}"] = round(value / peak, 4)

    for name, raw in raws.items():
        table, m = result[name]["prefill_kernels_ms"], raw["layers"][0]["mixer"]
        H, dq, vd, rank = m["heads"], m["dim"] + m["rot_dim"], m["vdim"], m["kv_rank"]

        def per_call(key):
            return table[key]["ms"] / table[key]["calls"] if key in table else None

        for key in ("latent_attention", "latent_unfolded_attention"):
            t = per_call(key)
            if t:   # scores and outputs over the visible pairs; the unfolded form also its up-projection
                flops = H * scored * 2 * ((dq + vd) if key != "latent_attention" else (2 * rank + m["rot_dim"]))
                put(f"{name}_{key}", (flops + (2 * tokens * rank * H * (m["dim"] + vd) if key != "latent_attention" else 0)) / t / 1e9,
                    pk["bf16_tflops"], "TFLOPs")
        t = per_call("attention_tc")
        if t:       # the tcgen05 kernel of the unfolded form alone
            put(f"{name}_attention_tc", H * scored * 2 * (dq + vd) / t / 1e9, pk["bf16_tflops"], "TFLOPs")
        t = per_call("routed_experts")
        if t:
            put(f"{name}_experts", pairs * (3 if name == "pafevik" else 2) * 2 * w * 1408 / t / 1e9, pk["bf16_tflops"], "TFLOPs")
        t = per_call("route")
        if t:
            roof[f"{name}_route_us"] = round(t * 1e3, 1)
        t = per_call("norm_stream")
        if t:       # Vesidra's norms also form the stream's last sum
            put(f"{name}_norm_stream", tokens * w * ((4 + 4 + 4 + 2) if name != "pafevik" else (4 + 2)) / t / 1e6, pk["hbm_gbs"], "GBps")
        t = per_call("add_stream")
        if t:
            put(f"{name}_add_stream", tokens * w * 12 / t / 1e6, pk["hbm_gbs"], "GBps")
        t = per_call("glu_act")
        if t:
            put(f"{name}_glu_act", tokens * 4 * w * 6 / t / 1e6, pk["hbm_gbs"], "GBps")
        t = table.get("matmul_nt")
        if t:       # all library products of the prompt but the head's (one row)
            if name == "pafevik":
                q = m["q_rank"] * (w + H * dq)
                flops = 2 * tokens * 4 * (q + w * (rank + m["rot_dim"] + H * vd) + w * H * vd + rank * H * (m["dim"] + vd))
            else:
                flops = 2 * tokens * (4 * (w * (H * dq + rank + m["rot_dim"] + H) + w * H * vd + rank * H * (m["dim"] + vd))
                                      + 2 * 3 * w * 4 * w + 2 * 2 * w * 2816)
            put(f"{name}_library_products", flops / t["ms"] / 1e9, pk["bf16_tflops"], "TFLOPs")
    result["roofline"] = roof
    result["peaks"] = pk
    print(json.dumps(result))
    return 0


# ---- Vabedra beside Figudra at equal size (`--only vabedra [--size s|m]`) ----
# Sizes that resemble a served model's layers: the width; four layers that take turns, an attention beside a delta rule (16
# or 32 heads of 128 on a quarter as many K/V heads with biases, normed and partly rotated queries and keys with frequencies
# scaled by wavelength, capped scores, a window of 1,024 that keeps the first 4 tokens and one added to the denominator; as
# many delta heads of 128 x 128 with a decay per key channel, decay and gate through ranks of 64, filters of 4 taps) and a
# delta rule alone (as many heads with one decay a head, two of them on a query/key head), each over 64 experts of 1,408 with
# clamped units of which a token uses 6, and a token input of 64 columns. Figudra beside it is `--only figudra`'s model of
# the same width, heads and experts: the library's other design with a state of 128 x 128 a head, a decay per key channel, a
# windowed attention that keeps the first tokens and gated experts.
def vabedra_config(size):
    z = PAFEVIK_SIZES[size]
    w, heads = z["width"], z["heads"]
    left = {"heads": heads, "kv_heads": heads // 4, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 30.0,
            "mask": {"size": 1024, "keep_first": 4},
            "rot": {"base": 10000.0, "dims": 64, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 2048}}}
    right = {"heads": heads, "kv_heads": heads, "dim": 128, "vdim": 128, "conv": 4, "rank": 64}
    alone = {"heads": heads, "kv_heads": heads // 2, "dim": 128, "vdim": 128, "conv": 4}
    moe = {"kind": "moe", "expert": {"ff": 1408, "limit": 7.0}, "router": {"experts": 64, "top": 6}}
    pair = {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": moe}
    return {"architecture": "Vabedra", "vocab": 32000, "width": w, "norm": {"eps": 1e-6}, "postln_alpha": 2.0,
            "embedding": {"scale": w ** 0.5}, "token_side": {"dim": 64},
            "layers": [pair, {"type": "delta", "mixer": alone, "mlp": moe}] * 2}


def run_vabedra(args):
    import torch

    import pytorch_transformers_b200 as ptb

    torch.cuda.set_device(0)
    pk = peaks()
    gen = torch.Generator().manual_seed(0)
    tokens, batch, context = args.prefill_tokens, args.batch, args.context
    raw, fig = vabedra_config(args.size), figudra_config(args.size)
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    left, right, w = raw["layers"][0]["mixer"]["left"], raw["layers"][0]["mixer"]["right"], raw["width"]
    result = {"only": "vabedra", "size": args.size, "prefill_tokens": tokens, "batch": batch, "context": context,
              "config": {"width": w, "layers": len(raw["layers"]), "heads": left["heads"]}}
    for name, cfg in (("vabedra", ptb.VabedraConfig.from_dict(raw)), ("figudra", ptb.FigudraConfig.from_dict(fig))):
        model = ptb.AutoModelForCausalLM.from_config(cfg, seed=0, dtype="bfloat16")
        result[name] = measure_prefill_and_decode(model, args, gen, flush)
        del model
        torch.cuda.empty_cache()
    V, F = result["vabedra"]["prefill_kernels_ms"], result["figudra"]["prefill_kernels_ms"]
    VD, FD = result["vabedra"]["decode_kernels_ms"], result["figudra"]["decode_kernels_ms"]

    def per_call(table, key):
        return table[key]["ms"] / table[key]["calls"] if key in table else None

    roof = {}

    def rate(name, t, flops=None, moved=None):
        """Achieved rates of a call of t ms against the measured peaks: operations, bytes or both."""
        if not t:
            return
        if flops is not None:
            roof[f"{name}_TFLOPs"] = round(flops / t / 1e9, 1)
            roof[f"{name}_frac_of_burst"] = round(flops / t / 1e9 / pk["bf16_tflops"], 4)
        if moved is not None:
            roof[f"{name}_GBps"] = round(moved / t / 1e6, 1)
            roof[f"{name}_frac_of_hbm"] = round(moved / t / 1e6 / pk["hbm_gbs"], 4)

    H, G, d, vd = left["heads"], left["kv_heads"], left["dim"], left["vdim"]
    keep, size = left["mask"]["keep_first"], left["mask"]["size"]
    seen = sum(min(t + 1, size) + max(0, min(keep, t + 1 - size)) for t in range(tokens))
    full = tokens * (tokens + 1) // 2
    rate("attention_prefill", per_call(V, "attention_mma"), flops=H * seen * 2 * (d + vd))
    if "attention_mma" in F:    # one windowed and one full layer share the table's row
        rate("figudra_attention_prefill", F["attention_mma"]["ms"], flops=H * (seen + full) * 2 * (d + vd))
    # the delta rule: queries, keys and values in, decays in (per channel in two layers, per head in two), float32 rows out;
    # what it needs a token and head: the read at the key, the write and the read at the query, 3 dim vdim multiply-adds
    lh, ld, lv = right["heads"], right["dim"], right["vdim"]
    io = tokens * lh * (2 * (2 * ld + lv) + (4 * ld + 4) / 2 + 4 * lv)
    rate("delta_rule_prefill", per_call(V, "delta_rule"), flops=lh * tokens * 2 * 3 * ld * lv, moved=io)
    rate("figudra_gla_prefill", per_call(F, "gla"), flops=lh * tokens * 2 * 3 * ld * lv, moved=tokens * lh * (2 * (2 * ld + lv) + 4 * ld + 4 * lv))
    # half of the calls form decays per channel (float32 in and out); half have two heads on a query/key head
    rate("delta_prepare_prefill", per_call(V, "delta_prepare"), moved=tokens * lh * (4 * (ld + ld / 2 + lv) + 8 * ld / 2))
    rate("figudra_gla_decay_prefill", per_call(F, "gla_decay_"), moved=tokens * lh * ld * 8)
    pairs = tokens * 6
    rate("expert_rows_prefill", per_call(V, "expert_rows"), flops=pairs * 3 * 2 * w * 1408)
    rate("figudra_expert_rows_prefill", per_call(F, "expert_rows"), flops=pairs * 3 * 2 * w * 1408)
    rate("post_norm_pair_prefill", per_call(V, "post_norm_pair"), moved=tokens * w * (4 * 4 + 2))
    rate("post_norm_prefill", per_call(V, "post_norm"), moved=tokens * w * (3 * 4 + 2))
    rate("post_norm_experts_prefill", per_call(V, "post_norm_experts"), moved=tokens * w * (2 * 4 + 6 * 4 + 2))
    rate("norm_add_prefill", per_call(V, "norm_add"), moved=tokens * w * (3 * 4 + 2))
    rate("figudra_norm_stream_prefill", per_call(F, "norm_stream"), moved=tokens * w * (4 + 4 + 4 + 2))
    rate("head_norm_gate_prefill", per_call(V, "head_norm_gate"), moved=tokens * lh * lv * (4 + 3 + 2))      # half of the gates float32
    rate("figudra_head_norm_gate_prefill", per_call(F, "head_norm_gate"), moved=tokens * lh * lv * (4 + 2 + 2))
    rows = tokens * ((H + G) * d + G * vd) * 4
    rate("rope_norm_store_prefill", per_call(V, "rope_norm_store"), moved=rows)
    rate("figudra_rope_norm_store_prefill", per_call(F, "rope_norm_store"), moved=rows)
    if "matmul_nt" in V:        # all library products of the prompt
        n_att = 2 * ((H + G) * d + G * vd + H * vd)
        n_pair = 2 * (2 * lh * ld + 2 * lh * lv + lh + 128)
        n_alone = 2 * (lh * ld + 3 * lh * lv + 2 * lh)
        flops = 2 * tokens * (w * (n_att + n_pair + n_alone) + 2 * 128 * lh * (ld + lv) + 4 * 2 * 64 * w)
        rate("library_products", V["matmul_nt"]["ms"], flops=flops)
    # single tokens, launched one by one: event pairs around small kernels hold the launch too
    state = batch * lh * ld * lv * 8
    rate("delta_rule_decode", per_call(VD, "delta_rule"), moved=state)
    rate("figudra_gla_decode", per_call(FD, "gla"), moved=state)
    result["roofline"] = roof
    result["peaks"] = pk
    print(json.dumps(result))
    return 0


def run_ours(args):
    if args.only == "vabedra":
        return run_vabedra(args)
    if args.only == "vesidra":
        return run_vesidra(args)
    if args.only == "figudra":
        return run_figudra(args)
    if args.only == "pafevik":
        return run_pafevik(args)
    if args.only == "pogezen":
        return run_pogezen(args)
    if args.only == "zalunex":
        return run_zalunex(args)
    if args.only == "sample":
        return run_sample(args)
    if args.only == "decode-attention":
        return run_decode_attention(args)
    if args.only == "prefill-attention":
        return run_prefill_attention(args)
    if args.only == "mma-cadence":
        return run_mma_cadence(args)
    if args.only == "linear":
        return run_linear(args)
    if args.only == "fill":
        return run_fill(args)
    import torch

    import pytorch_transformers_b200 as ptb
    from pytorch_transformers_b200 import kernels
    from pytorch_transformers_b200.config.generation import GenerationConfig
    from pytorch_transformers_b200.sampling import DeviceSelector

    torch.cuda.set_device(0)
    shape = SHAPES[args.shape]
    layers = args.layers or shape["num_hidden_layers"]
    cfg = ptb.FalconConfig.from_dict(dict(shape, num_hidden_layers=layers))
    model = ptb.AutoModelForCausalLM.from_config(cfg, seed=0, dtype="bfloat16", device="cuda:0")
    pk = peaks()
    gen = torch.Generator().manual_seed(0)

    def prompts(n, length):
        return torch.randint(0, cfg.vocab_size, (n, length), generator=gen).tolist()

    def decode_run(batch, steps, warmup, sample_clocks=False, context=CONTEXT):
        """Prefill `batch` prompts of `context` tokens, then time `steps` decode steps."""
        CONTEXT = context
        total = CONTEXT + SETTLE_STEPS + steps + warmup + 1
        cache = model.new_cache(batch * ((total + 63) // 64 * 64))
        slots = [cache.open() for _ in range(batch)]
        opts = GenerationConfig(do_sample=False)
        sel = DeviceSelector(kernels, model.device, cfg.vocab_size, opts, max_rows=batch)
        ps = prompts(batch, CONTEXT)
        chunk = max(1, 8192 // CONTEXT)                      # prompts go in a few at a time to bound activations
        for i in range(0, batch, chunk):
            logits = model.step(cache, slots[i:i + chunk], ps[i:i + chunk], want="last")
        logits = model.step(cache, slots, [[1]] * batch, want="last")
        ids = list(range(batch))

        def one():
            # one decode step as the generation loop runs it: the selection runs on the device, meanwhile
            # the host builds the next step and launches it with the tokens still on the device, then
            # reads the tokens (steps that cannot be launched ahead wait for the tokens first)
            nonlocal logits
            pending = sel.begin(logits, ids, 0)
            model.prepare_next(cache, slots)
            ahead = model.step_ahead(cache, slots, sel.device_tokens(pending))
            toks = sel.finish(pending)
            logits = ahead if ahead is not None else model.step(cache, slots, [[t] for t in toks], want="last")

        for _ in range(SETTLE_STEPS + warmup):
            one()
        torch.cuda.synchronize()
        sampler = ClockSampler() if sample_clocks else None
        l0 = kernels.launches
        if sampler:
            sampler.__enter__()
        start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        torch.cuda.profiler.start()   # a profiler started with --profile-from-start off sees the timed steps only
        start.record()
        for _ in range(steps):
            one()
        end.record()
        torch.cuda.synchronize()
        torch.cuda.profiler.stop()
        if sampler:
            sampler.__exit__()
        ms = start.elapsed_time(end) / steps
        launches = kernels.launches - l0
        ctx_mid = CONTEXT + 1 + SETTLE_STEPS + warmup + steps / 2
        cache.close_all()
        del cache
        torch.cuda.empty_cache()
        return ms, launches, ctx_mid, (sampler.summary() if sampler else None)

    if args.no_graphs:
        model.use_graphs = False
    if args.only == "config":
        return run_config(args, model, cfg, layers, pk)
    if args.only == "decode":
        ms, launches, ctx_mid, _ = decode_run(args.batch, args.steps, args.warmup, context=args.context)
        kv_bytes = args.batch * ctx_mid * layers * 2 * cfg.kv_heads_eff * cfg.head_dim * 2
        print(json.dumps({"only": "decode", "shape": args.shape, "batch": args.batch, "context": args.context,
                          "layers": layers,
                          "ms_per_step": round(ms, 4), "launches_per_step": launches / args.steps,
                          "GBps": round((model.weight_bytes() - (0 if cfg.tie_word_embeddings else
                                                                cfg.vocab_size * cfg.hidden_size * 2) + kv_bytes)
                                        / ms / 1e6, 1)}))
        return 0

    # ---- prefill of 2,048 tokens (one prompt) ----
    n_prefill = args.prefill_tokens if args.only == "prefill" else PREFILL_TOKENS
    cache = model.new_cache(n_prefill + 64)
    p = prompts(1, n_prefill)
    times = []
    for i in range(2 + 3):
        s = cache.open()
        torch.cuda.synchronize()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        model.step(cache, [s], p, want="last")
        b.record()
        torch.cuda.synchronize()
        if i >= 2:
            times.append(a.elapsed_time(b))
        cache.close(s)
    del cache
    pre_ms = statistics.median(times)
    if args.only == "prefill":
        print(json.dumps({"only": "prefill", "shape": args.shape, "tokens": n_prefill, "layers": layers,
                          "ms": round(pre_ms, 3),
                          "TFLOPs": round(prefill_flops(shape, layers, n_prefill) / pre_ms / 1e9, 1)}))
        return 0
    pre_flops = prefill_flops(FALCON_7B, layers, PREFILL_TOKENS)
    prefill = {"value": round(PREFILL_TOKENS / pre_ms * 1e3, 1), "tokens": PREFILL_TOKENS, "ms": round(pre_ms, 3),
               "frac": round(pre_flops / (pre_ms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4),
               "frac_sustained": round(pre_flops / (pre_ms * 1e-3) / (pk["bf16_tflops_sustained"] * 1e12), 4)}

    # ---- headline: decode at batch 8 ----
    batch = args.batch
    ms, launches, ctx_mid, clocks = decode_run(batch, args.steps, args.warmup, sample_clocks=True)
    value = batch / ms * 1e3
    need = decode_bytes(FALCON_7B, layers, batch, ctx_mid)
    achieved = need / (ms * 1e-3) / 1e9
    roofline = {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                "frac": round(achieved / pk["hbm_gbs"], 4), "peaks": pk["source"]}

    points, points_roofline = {}, {}
    for b in (1, 64):
        pms, _, pctx, _ = decode_run(b, max(8, args.steps // 2), 3)
        points[f"decode_b{b}"] = round(b / pms * 1e3, 1)
        pbytes = decode_bytes(FALCON_7B, layers, b, pctx)
        points_roofline[f"decode_b{b}"] = {"ms_per_step": round(pms, 4), "bytes": int(pbytes),
                                           "achieved": round(pbytes / (pms * 1e-3) / 1e9, 1),
                                           "frac": round(pbytes / (pms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}

    # ---- end to end through generate(): host token lists in, host token lists out ----
    # After the prefill (seconds of tensor-core work under the power cap) the device runs its first tens of
    # decode steps 5 to 10 % slower and comes back in stages; SETTLE_STEPS untimed steps come before the W
    # warm-up steps so that the K timed steps measure decoding, not the prefill's aftermath.
    n_new = SETTLE_STEPS + args.warmup + args.steps
    ps = prompts(batch, CONTEXT)
    stamps = []
    model.generate(ps, max_new_tokens=2, eos_token_id=None, max_batch_size=batch)       # sizes the cache, warms up
    t_prefill_done = [None]

    def on_token(r, tok):
        if r == batch - 1:
            stamps.append(time.perf_counter())

    torch.cuda.synchronize()
    model.generate(ps, max_new_tokens=n_new, eos_token_id=None, max_batch_size=batch, on_token=on_token)
    torch.cuda.synchronize()
    t_end = time.perf_counter()
    # stamps[i] is taken when step i's tokens have reached the host; steps after the warm-up count
    e2e_s = (stamps[-1] - stamps[-1 - args.steps]) / args.steps
    e2e = {"value": round(batch / e2e_s, 1), "unit": "tokens/s", "settle_steps": SETTLE_STEPS,
           "h2d_bytes_per_step": int(model.last_h2d_bytes),
           "d2h_bytes_per_step": 4 * batch}

    out = {
        "metric": "decode tokens/s, Falcon-7B shape, bf16, batch 8, context 2048", "value": round(value, 1),
        "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup, "ms_per_step": round(ms, 4),
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
        "impl": "ours",
        "config": workload_config(layers, batch),
        "notes": {"sampling": "greedy, on the device", "cache_page": 64, "decode_steps": "CUDA graphs",
                  "timing": "CUDA events around K steps", "settle_steps": SETTLE_STEPS,
                  "settle": "untimed decode steps after every prefill, before the W warm-up steps"},
        "prefill": prefill, "roofline": roofline, "points": points, "points_roofline": points_roofline, "e2e": e2e,
        "gpu_launches": launches,
        "clocks": clocks,
    }
    print(json.dumps(out), flush=True)
    return 0


def run_reference(args):
    """The reference's own FalconForCausalLM.generate (bf16, its default attention path, its
    DynamicCache) from baseline/_ref, same shapes, random weights, same metric."""
    ref = os.path.join(ROOT, "baseline", "_ref")
    if not os.path.isdir(os.path.join(ref, "transformers")):
        print(json.dumps({"impl": "reference", "unavailable": "baseline/_ref holds no installed reference"}))
        return 0
    try:
        import importlib.metadata as md
        os.environ["HF_HUB_OFFLINE"] = "1"
        os.environ["TRANSFORMERS_OFFLINE"] = "1"
        sys.path.insert(0, ref)
        real = md.version
        # the reference checks two wheels' versions at import; answer with versions in its range
        md.version = lambda n: {"tokenizers": "0.21.4", "huggingface-hub": "0.30.0"}.get(
            n.lower().replace("_", "-")) or real(n)
        import torch
        from transformers import FalconConfig, FalconForCausalLM
        torch.cuda.set_device(0)
        layers = args.layers or FALCON_7B["num_hidden_layers"]
        cfg = FalconConfig(**dict(FALCON_7B, num_hidden_layers=layers))
        torch.manual_seed(0)
        with torch.device("cuda:0"):
            model = FalconForCausalLM(cfg).to(torch.bfloat16).eval()
        batch = args.batch
        ids = torch.randint(0, cfg.vocab_size, (batch, CONTEXT), generator=torch.Generator().manual_seed(0))
        pinned = ids.pin_memory()
        stamps = []

        class Stamp:
            def put(self, value):
                value.cpu() if hasattr(value, "cpu") else None
                stamps.append(time.perf_counter())

            def end(self):
                pass

        def run(n_new, streamer=None):
            dev = pinned.to("cuda:0", non_blocking=True)
            return model.generate(dev, attention_mask=torch.ones_like(dev), max_new_tokens=n_new, do_sample=False,
                                  eos_token_id=None, pad_token_id=0, streamer=streamer)

        # device-timed decode: (prefill + W+K tokens) - (prefill + W tokens), CUDA events
        def timed(n_new):
            torch.cuda.synchronize()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            run(n_new)
            b.record()
            torch.cuda.synchronize()
            return a.elapsed_time(b)

        timed(2)
        sampler = ClockSampler()
        with sampler:
            t_short = timed(args.warmup)
            t_long = timed(args.warmup + args.steps)
        ms = (t_long - t_short) / args.steps
        # end to end: wall clock between tokens reaching the host, warm-up steps dropped
        # (generate() batch > 1 cannot stream through TextStreamer; a plain streamer object serves)
        stamps.clear()
        try:
            run(args.warmup + args.steps, streamer=Stamp())
            per = (stamps[-1] - stamps[args.warmup]) / (len(stamps) - 1 - args.warmup)
            e2e = {"value": round(batch / per, 1), "unit": "tokens/s", "h2d_bytes_per_step": 0,
                   "d2h_bytes_per_step": 8 * batch}
        except Exception as e:  # noqa: BLE001
            e2e = {"value": None, "unit": "tokens/s", "error": str(e)[:200]}
        out = {"metric": "decode tokens/s, Falcon-7B shape, bf16, batch 8, context 2048", "impl": "reference",
               "value": round(batch / ms * 1e3, 1), "unit": "tokens/s", "n_gpus": 1, "steps": args.steps,
               "warmup": args.warmup, "ms_per_step": round(ms, 4), "higher_is_better": True, "scaling": "weak",
               "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
               "config": workload_config(layers, batch),
               "notes": {"sampling": "greedy", "attention": "sdpa (reference default)", "cache": "DynamicCache",
                         "timing": "generate(W+K) minus generate(W), CUDA events"},
               "e2e": e2e, "gpu_launches": 0, "clocks": sampler.summary()}
        print(json.dumps(out), flush=True)
    except Exception as e:  # noqa: BLE001
        print(json.dumps({"impl": "reference", "unavailable": f"{type(e).__name__}: {str(e)[:300]}"}))
    return 0


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=5)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--layers", type=int, default=0, help="fewer layers than the configuration's (0: all)")
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--only", default="", choices=["", "decode", "prefill", "sample", "decode-attention", "prefill-attention", "config", "linear",
                             "fill", "mma-cadence", "pafevik", "zalunex", "pogezen", "figudra", "vesidra", "vabedra"],
                    help="run one section only and print its numbers (for profilers)")
    ap.add_argument("--shape", default="7b", choices=sorted(SHAPES), help="model shape for --only decode / prefill")
    ap.add_argument("--size", default="s", choices=sorted(PAFEVIK_SIZES), help="layer sizes for --only pafevik, --only zalunex, --only pogezen, --only figudra, --only vesidra and --only vabedra")
    ap.add_argument("--prefill-tokens", type=int, default=PREFILL_TOKENS, help="prompt length for --only prefill")
    ap.add_argument("--context", type=int, default=CONTEXT, help="cached tokens per sequence for --only decode")
    ap.add_argument("--past", type=int, default=0, help="cached tokens before the prompt for --only prefill-attention")
    ap.add_argument("--rows", type=int, default=8, help="rows of the activation for --only linear")
    ap.add_argument("--decode-steps", type=int, default=0,
                    help="decode steps of --only config (0: the number BASELINE gives for the shape)")
    ap.add_argument("--settle", type=int, default=SETTLE_STEPS,
                    help="untimed decode steps after a prefill, before the warm-up steps (0 for profiler runs)")
    ap.add_argument("--no-graphs", action="store_true", help="launch every kernel of a decode step itself")
    args = ap.parse_args()
    globals()["SETTLE_STEPS"] = max(0, args.settle)
    if args.gpus != 1:
        print(f"bench.py measures one GPU: this library is a single-GPU engine, --gpus {args.gpus} is not run")
        return 2
    args.warmup = max(3, args.warmup)
    if (args.shape != "7b" or args.prefill_tokens != PREFILL_TOKENS or args.context != CONTEXT) and not args.only:
        print("--shape, --context and --prefill-tokens go with --only decode / --only prefill (the headline is measured on "
              "the 7B shape with a prefill of 2,048 tokens)")
        return 2
    if args.only == "config" and args.shape not in BASELINE_RUNS:
        print("--only config runs BASELINE's configurations of the larger shapes: --shape 11b or --shape 40b")
        return 2
    if args.impl == "reference":
        return run_reference(args)
    return run_ours(args)


if __name__ == "__main__":
    sys.exit(main())
