#!/usr/bin/env python3
"""Decode and prefill throughput of the engine at Llama-3.2-1B size, one GPU.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--batch 8] [--layers L]

A "step" is one decode step of ``--batch`` requests.  Each request is a 512-token
uniform-random prompt; after the prompts are read, W decode steps warm up and
exactly K are timed, once on the device (CUDA events on the launching stream:
``value``) and once end to end through the Python entry point (host token ids in,
sampled ids out at every step: ``e2e``).  Weights are random (N(0, 0.02), norms
1 + N(0, 0.02)), bfloat16, 16-token pages, context limit 4096.  One JSON line goes
to standard output; progress goes to standard error.
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

LLAMA_1B = {
    "architectures": ["LlamaForCausalLM"], "model_type": "llama",
    "vocab_size": 128256, "hidden_size": 2048, "intermediate_size": 8192, "num_hidden_layers": 16,
    "num_attention_heads": 32, "num_key_value_heads": 8, "head_dim": 64,
    "rms_norm_eps": 1e-5, "rope_theta": 500000.0,
    "rope_scaling": {"rope_type": "llama3", "factor": 32.0, "low_freq_factor": 1.0,
                     "high_freq_factor": 4.0, "original_max_position_embeddings": 8192},
    "max_position_embeddings": 131072, "tie_word_embeddings": True, "hidden_act": "silu",
}
_LLAMA3_ROPE = {"rope_type": "llama3", "low_freq_factor": 1.0, "high_freq_factor": 4.0,
                "original_max_position_embeddings": 8192}
LLAMA_3B = dict(LLAMA_1B, hidden_size=3072, num_hidden_layers=28, num_attention_heads=24, num_key_value_heads=8,
                head_dim=128, intermediate_size=8192, rope_scaling=dict(_LLAMA3_ROPE, factor=32.0))
LLAMA_8B = dict(LLAMA_1B, hidden_size=4096, num_hidden_layers=32, num_attention_heads=32, num_key_value_heads=8,
                head_dim=128, intermediate_size=14336, tie_word_embeddings=False,
                rope_scaling=dict(_LLAMA3_ROPE, factor=8.0))
# The two serving workloads beside the headline: continuous batching under Poisson arrivals at the
# 3B shape, and 64 long requests at the 8B shape in a pool that cannot hold them all.
WORKLOADS = {
    "serve3b": {"model": LLAMA_3B, "name": "Llama-3.2-3B shape", "requests": 256, "prompt_len": (128, 2048),
                "output_len": (64, 512), "arrival_rate": 64.0, "context_len": 8192, "max_num_seqs": 256,
                "pool_fraction_of_need": 0.6},
    "stress8b": {"model": LLAMA_8B, "name": "Llama-3.1-8B shape", "requests": 64, "prompt_len": (4096, 4096),
                 "output_len": (512, 512), "arrival_rate": 0.0, "context_len": 16384, "max_num_seqs": 64,
                 "pool_fraction_of_need": 0.75},
}
FULL_LAYERS = LLAMA_1B["num_hidden_layers"]
CONTEXT_LEN = 4096
PROMPT_LEN = 512
NEW_TOKENS = 256
PREFILL_TOKENS = 2048
PAGE_SIZE = 16
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


def log(msg):
    print(f"[bench] {msg}", file=sys.stderr, flush=True)


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        try:
            d = json.load(open(path))
            out = {"hbm_gbs": float(d["hbm_gbs"]), "bf16_tflops": float(d["bf16_tflops"]), "source": "measured"}
            if "bf16_tflops_sustained" in d:
                out["bf16_tflops_sustained"] = float(d["bf16_tflops_sustained"])
            return out
        except Exception as e:  # an unreadable file must not cost the run
            log(f"MEASURED_PEAKS.json could not be used ({e}); falling back")
    return dict(FALLBACK_PEAKS)


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while a region runs."""
    FIELDS = ("clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.hw_slowdown,"
              "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
              "clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.proc, self.lines = None, []

    def start(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", "-i", "0", f"--query-gpu={self.FIELDS}", "--format=csv,noheader,nounits", "-lms", "100"],
                stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            self.thread = threading.Thread(target=self._read, daemon=True)
            self.thread.start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.lines.append((time.perf_counter(), line.strip()))

    def stop(self):
        if self.proc is not None:
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()

    def summary(self, windows):
        """Clocks of the samples that fall inside the timed windows [(t0, t1), ...]."""
        sm, mx, reasons = [], [], set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        inside = [(t, line) for t, line in self.lines if any(a <= t <= b for a, b in windows)]
        if len(inside) < 3:
            # timed regions shorter than the sampling period: take the samples next to them as well
            inside = [(t, line) for t, line in self.lines if any(a - 0.25 <= t <= b + 0.25 for a, b in windows)]
        for t, line in inside:
            parts = [p.strip() for p in line.split(",")]
            if len(parts) < 7:
                continue
            try:
                sm.append(float(parts[0]))
                mx.append(float(parts[1]))
            except ValueError:
                continue
            for name, val in zip(names, parts[3:7]):
                if val.lower().startswith("active"):
                    reasons.add(name)
        if not sm:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": [], "samples": 0}
        return {"sm_mhz": statistics.median(sm), "sm_max_mhz": max(mx), "reasons": sorted(reasons),
                "samples": len(sm)}


def model_numbers(cfg, layers):
    """Bytes and FLOPs of this model's steps, from the configuration."""
    H, I, V = cfg["hidden_size"], cfg["intermediate_size"], cfg["vocab_size"]
    nq, nkv, d = cfg["num_attention_heads"], cfg["num_key_value_heads"], cfg["head_dim"]
    layer_matrix = (nq * d + 2 * nkv * d) * H + H * nq * d + 3 * I * H
    weight_elems = layers * (layer_matrix + 2 * H) + V * H + H
    return {
        "weight_bytes": 2 * weight_elems,                   # bfloat16, every weight read once per step
        "kv_bytes_per_token": layers * 2 * nkv * d * 2,      # keys and values, bfloat16
        "layer_matrix_elems": layer_matrix,
        "attn_flops_per_pair": 4 * nq * d,                   # q.k and p.v per (query, key) pair, all heads
    }


def prefill_flops(cfg, layers, T):
    n = model_numbers(cfg, layers)
    gemm = 2 * T * layers * n["layer_matrix_elems"] + 2 * cfg["vocab_size"] * cfg["hidden_size"]
    attn = layers * n["attn_flops_per_pair"] * T * (T + 1) // 2
    return gemm + attn


def run_decode(llm, batch, steps, warmup, end_to_end, seed):
    """Reads ``batch`` prompts, warms up, times ``steps`` decode steps.  Returns
    (seconds, mean context during the timed steps, launches, (t0, t1) wall window)."""
    import numpy as np
    import torch
    from kv_cache_optimization_for_llm_b200 import SamplingParams, ops
    eng = llm.engine
    rng = np.random.default_rng(seed)
    vocab = eng.runner.vocab_size
    sp = SamplingParams(max_tokens=NEW_TOKENS, ignore_eos=True)
    ids = [eng.add_request(rng.integers(0, vocab, PROMPT_LEN).tolist(), sp) for _ in range(batch)]
    produced = {i: 0 for i in ids}
    while min(produced.values()) < 1:          # read the prompts (mixed steps until every request decodes)
        for ev in eng.step():
            if ev.token is not None:
                produced[ev.request_id] += 1
    lead = max(produced.values())
    # Warm-up: steps of single tokens only (the timed kind), at least three even when some
    # requests already decoded while others still read their prompts.
    for _ in range(max(3, warmup - (lead - 1))):
        eng.step()
        lead += 1
    if lead + steps > NEW_TOKENS:
        raise SystemExit(f"{lead} tokens were produced before timing; {steps} more exceed the budget of {NEW_TOKENS}")
    torch.cuda.synchronize()
    ctx0 = PROMPT_LEN + max(len(eng.output(i)) for i in ids)
    launches0 = ops.launch_count + eng.runner.graph_launches
    start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    w0 = time.perf_counter()
    start.record()
    n_tok = 0
    for _ in range(steps):
        n_tok += sum(1 for ev in eng.step() if ev.token is not None)
    stop.record()
    torch.cuda.synchronize()
    w1 = time.perf_counter()
    assert n_tok == batch * steps, f"{n_tok} tokens from {batch} requests in {steps} steps"
    launches = ops.launch_count + eng.runner.graph_launches - launches0
    seconds = (w1 - w0) if end_to_end else start.elapsed_time(stop) / 1000.0
    run_decode.h2d_bytes = eng.runner.builder.last_h2d_bytes      # of one decode step of this batch
    for i in ids:
        eng.abort(i)
    assert eng.runner.manager.check() == "" and eng.runner.manager.live_requests() == 0
    return seconds, ctx0 + (steps - 1) / 2.0, launches, (w0, w1)


def run_prefill(llm, reps, warmup, seed):
    import numpy as np
    import torch
    from kv_cache_optimization_for_llm_b200.engine.batch import StepEntry
    r = llm.engine.runner
    rng = np.random.default_rng(seed)
    toks = rng.integers(0, r.vocab_size, PREFILL_TOKENS).tolist()
    times = []
    for k in range(warmup + reps):
        rid = 10_000_000 + k
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        start.record()
        logits = r.step([StepEntry(rid, toks, 0, [PREFILL_TOKENS - 1])])
        stop.record()
        torch.cuda.synchronize()
        assert logits.shape == (1, r.vocab_size)
        r.release(rid)
        if k >= warmup:
            times.append(start.elapsed_time(stop))
    return statistics.median(times)


def run_first_token(llm, prompt_len, reps, warmup, seed):
    """Milliseconds from handing one prompt of ``prompt_len`` tokens to an idle engine to its first
    token on the host, through add_request and step (median)."""
    import numpy as np
    import torch
    from kv_cache_optimization_for_llm_b200 import SamplingParams
    eng = llm.engine
    rng = np.random.default_rng(seed)
    times = []
    for k in range(warmup + reps):
        prompt = rng.integers(0, eng.runner.vocab_size, prompt_len).tolist()
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        rid = eng.add_request(prompt, SamplingParams(max_tokens=2, ignore_eos=True))
        first = None
        while first is None:
            for ev in eng.step():
                if ev.request_id == rid and ev.token is not None and first is None:
                    first = time.perf_counter()
        while eng.has_unfinished():
            eng.step()
        if k >= warmup:
            times.append((first - t0) * 1e3)
    return statistics.median(times)


def run_value_check(cfg, layers=2):
    """The numbers behind the timings: a model of the benchmark's widths with ``layers`` layers is written to a
    temporary folder and its logits, on the paths that the benchmark times (one 2048-token portion; eight
    requests decoding beside each other from 512-token prompts, replayed from a captured graph), are compared
    with the plain implementation under tests/ at the limit the tests use for bfloat16."""
    import shutil
    import tempfile

    import numpy as np

    sys.path.insert(0, os.path.join(ROOT, "tests"))
    import plain_llama as P
    from kv_cache_optimization_for_llm_b200 import EngineConfig
    from kv_cache_optimization_for_llm_b200.engine.batch import StepEntry
    from kv_cache_optimization_for_llm_b200.engine.runner import ModelRunner
    from kv_cache_optimization_for_llm_b200.weights import write_random_model

    limit = 4e-2
    small = dict(cfg)
    small["num_hidden_layers"] = layers
    d = tempfile.mkdtemp(prefix="kvb200_bench_check_")
    try:
        write_random_model(d, small, seed=0, std=0.02, storage_dtype="bfloat16")
        pcfg, w = P.read_model_dir(d)
        r = ModelRunner(d, EngineConfig(dtype="bfloat16", page_size=PAGE_SIZE, num_pages=8 * 40 + 140, max_num_seqs=8,
                                        max_num_batched_tokens=PREFILL_TOKENS, max_model_len=CONTEXT_LEN))
        rng = np.random.default_rng(5)
        worst = {}

        def err(got, ref):
            return float(np.abs(got.astype(np.float64) - ref).max() / np.abs(ref).max())

        seq = rng.integers(0, cfg["vocab_size"], PREFILL_TOKENS).tolist()
        rows = [0, 777, PREFILL_TOKENS - 1]
        got = r.step([StepEntry(999, seq, 0, rows)]).float().cpu().numpy()
        r.release(999)
        worst["prefill_2048"] = err(got, P.forward(pcfg, w, seq, rows=rows))
        seqs = [rng.integers(0, cfg["vocab_size"], PROMPT_LEN + 3).tolist() for _ in range(8)]
        r.step([StepEntry(i, s_[:PROMPT_LEN], 0, []) for i, s_ in enumerate(seqs)][:4])
        r.step([StepEntry(i, s_[:PROMPT_LEN], 0, []) for i, s_ in enumerate(seqs)][4:])
        got = None
        for t in range(PROMPT_LEN, PROMPT_LEN + 3):
            got = r.step([StepEntry(i, [s_[t]], t, [0]) for i, s_ in enumerate(seqs)]).float().cpu().numpy()
        ref = np.stack([P.forward(pcfg, w, s_, rows=[PROMPT_LEN + 2])[0] for s_ in seqs])
        worst["decode_b8"] = err(got, ref)
        kinds = dict(r.step_kinds)
    finally:
        shutil.rmtree(d, ignore_errors=True)
    ok = all(v < limit for v in worst.values())
    return {"ok": ok, "limit": limit, "layers": layers, "worst_relative_error": {k: round(v, 5) for k, v in worst.items()},
            "step_kinds": kinds}


def _pct(xs, p):
    xs = sorted(xs)
    return xs[min(len(xs) - 1, int(round(p / 100.0 * (len(xs) - 1))))] if xs else None


def run_workload(name, seed=0):
    """One of WORKLOADS through the engine's own entry points (add_request, step), requests arriving
    in real time.  Every request must emit exactly its budget and no page may be lost; returns
    output tokens a second, time to the first token and time per further token, and what the
    scheduler had to drop and recompute."""
    import gc
    import numpy as np
    import torch
    from kv_cache_optimization_for_llm_b200 import LLM, SamplingParams
    wl = WORKLOADS[name]
    cfg = dict(wl["model"])
    rng = np.random.default_rng(seed)
    n = wl["requests"]
    p_len = rng.integers(wl["prompt_len"][0], wl["prompt_len"][1] + 1, n)
    o_len = rng.integers(wl["output_len"][0], wl["output_len"][1] + 1, n)
    gaps = rng.exponential(1.0 / wl["arrival_rate"], n) if wl["arrival_rate"] > 0 else np.zeros(n)
    arrive = np.cumsum(gaps) - gaps[0]
    need_tokens = int((p_len + o_len).sum())
    pool_tokens = int(need_tokens * wl["pool_fraction_of_need"])
    num_pages = max(pool_tokens // PAGE_SIZE, (int((p_len + o_len).max()) + PAGE_SIZE) // PAGE_SIZE + 1)
    log(f"{name}: building {wl['name']}, {cfg['num_hidden_layers']} layers, pool of {num_pages} pages "
        f"({num_pages * PAGE_SIZE} tokens; all requests together need {need_tokens})")
    llm = LLM.from_random(cfg, seed=0, std=0.02, dtype="bfloat16", page_size=PAGE_SIZE, num_pages=num_pages,
                          max_num_seqs=wl["max_num_seqs"], max_num_batched_tokens=PREFILL_TOKENS,
                          max_model_len=wl["context_len"], capture_graphs_at_start=True)
    eng = llm.engine
    kv_bytes = eng.runner.cache.bytes_per_page() * num_pages
    prompts = [rng.integers(0, cfg["vocab_size"], int(k)).tolist() for k in p_len]
    # warm-up: a prompt of two portions and a few decode steps (kernels loaded, allocator warm)
    eng.generate([prompts[0][:128] * 20], SamplingParams(max_tokens=4, ignore_eos=True))
    torch.cuda.synchronize()
    first, last, count = {}, {}, {i: 0 for i in range(n)}
    errors = []
    nxt = 0
    t0 = time.perf_counter()
    while nxt < n or eng.has_unfinished():
        now = time.perf_counter() - t0
        while nxt < n and arrive[nxt] <= now:
            eng.add_request(prompts[nxt], SamplingParams(max_tokens=int(o_len[nxt]), ignore_eos=True), request_id=1000 + nxt)
            nxt += 1
        if not eng.has_unfinished():
            time.sleep(max(0.0, min(0.001, arrive[nxt] - now)))
            continue
        for ev in eng.step():
            t = time.perf_counter() - t0
            i = ev.request_id - 1000
            if ev.token is not None:
                count[i] += 1
                first.setdefault(i, t)
                last[i] = t
            if ev.finished and ev.reason != "length":
                errors.append((i, ev.reason))
    torch.cuda.synchronize()
    seconds = time.perf_counter() - t0
    st = eng.stats()
    wrong = [i for i in range(n) if count[i] != int(o_len[i])]
    assert not errors and not wrong, f"{name}: requests ended early {errors[:3]} or with other counts than their budget {wrong[:3]}"
    assert eng.runner.manager.check() == "" and st["free_pages"] == [num_pages], "a page was lost"
    ttft = [1000.0 * (first[i] - arrive[i]) for i in range(n)]
    tpot = [1000.0 * (last[i] - first[i]) / (count[i] - 1) for i in range(n) if count[i] > 1]
    out_tokens = int(o_len.sum())
    res = {
        "value": round(out_tokens / seconds, 1), "unit": "output tokens/s", "seconds": round(seconds, 3),
        "requests": n, "prompt_tokens": int(p_len.sum()), "output_tokens": out_tokens,
        "total_tokens_per_s": round((out_tokens + int(p_len.sum())) / seconds, 1),
        "ttft_ms": {"p50": round(_pct(ttft, 50), 2), "p99": round(_pct(ttft, 99), 2)},
        "per_token_ms": {"p50": round(_pct(tpot, 50), 3), "p99": round(_pct(tpot, 99), 3)},
        "steps": int(st["steps"]), "preemptions": int(st["preemptions"]), "recomputed_tokens": int(st["recomputed_tokens"]),
        "step_kinds": st.get("step_kinds"),
        "config": {"model": wl["name"], "layers": cfg["num_hidden_layers"], "hidden_size": cfg["hidden_size"],
                   "heads": f"{cfg['num_attention_heads']}/{cfg['num_key_value_heads']}", "head_dim": cfg["head_dim"],
                   "intermediate_size": cfg["intermediate_size"], "tied_lm_head": bool(cfg["tie_word_embeddings"]),
                   "prompt_len": list(wl["prompt_len"]), "output_len": list(wl["output_len"]),
                   "arrivals": f"Poisson, {wl['arrival_rate']}/s" if wl["arrival_rate"] > 0 else "all at once",
                   "context_len": wl["context_len"], "page_size": PAGE_SIZE, "max_num_seqs": wl["max_num_seqs"],
                   "tokens_per_step": PREFILL_TOKENS, "pool_pages": num_pages, "pool_gb": round(kv_bytes / 1e9, 2),
                   "all_resident_gb": round(kv_bytes / num_pages / PAGE_SIZE * need_tokens / 1e9, 2), "seed": seed},
    }
    log(f"  {res['value']:.0f} output tok/s in {seconds:.2f} s, {st['steps']} steps, TTFT p50 {res['ttft_ms']['p50']:.0f} ms, "
        f"per token p50 {res['per_token_ms']['p50']:.2f} ms, {st['preemptions']} preemptions "
        f"({st['recomputed_tokens']} tokens recomputed)")
    del eng, llm
    gc.collect()
    torch.cuda.empty_cache()
    return res


# ---------------------------------------------------------------------------------------------
# Two designs at equal size (bench.py --compare <size>)
# ---------------------------------------------------------------------------------------------
COMPARE_SIZES = {
    # width, feed-forward, vocabulary, layers; heads of 64 for Llama and the delta-rule mixers; the latent attention
    # with heads of dim + rot and a latent of four value heads' width
    "w1024": dict(width=1024, ff=4096, vocab=32768, layers=6, heads=16, lat_heads=8, lat_dim=64, lat_rot=32, lat_vdim=64,
                  q_rank=384, kv_rank=256, low_rank=64),
    "w2048": dict(width=2048, ff=8192, vocab=32768, layers=6, heads=32, lat_heads=16, lat_dim=128, lat_rot=64,
                  lat_vdim=128, q_rank=768, kv_rank=512, low_rank=64),
}
FP32_FMA_TFLOPS_NOMINAL = 75.0    # 148 SMs x 128 lanes x 2 x ~1.97 GHz: no measured figure for the CUDA cores is at hand


def rezusun_config(z):
    mlp = {"kind": "dense", "ff": z["ff"]}
    general = {"type": "general_delta", "mixer": {"heads": z["heads"], "dim": 64, "decay_rank": z["low_rank"]}, "mlp": mlp}
    channel = {"type": "channel_delta", "mixer": {"heads": z["heads"], "kv_heads": z["heads"] // 4, "dim": 64, "vdim": 64,
                                                 "conv": 4, "decay_rank": z["low_rank"], "gate_rank": z["low_rank"]}, "mlp": mlp}
    latent = {"type": "latent_attention", "mlp": mlp, "mixer": {
        "heads": z["lat_heads"], "dim": z["lat_dim"], "rot_dim": z["lat_rot"], "vdim": z["lat_vdim"], "q_rank": z["q_rank"],
        "kv_rank": z["kv_rank"], "scale": (z["lat_dim"] + z["lat_rot"]) ** -0.5, "rot": {"base": 10000.0, "dims": z["lat_rot"]}}}
    return {"architecture": "Rezusun", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
            "layers": [[general, channel, latent][i % 3] for i in range(z["layers"])], "loop": None,
            "max_position_embeddings": CONTEXT_LEN}


def solulix_config(z, window=1024, keep_first=64, experts=True):
    """Six layers at the comparison's sizes: attention (heads of 64, a quarter as many key/value heads, four taps, a
    window of 1024 tokens that keeps the first 64) and the gated delta rule (heads of 64 x 64) in turn; dense
    feed-forwards of the same width as Llama's, and on every third layer 32 experts of a sixteenth of that width of
    which a token uses four, one identity expert and a shared expert of a quarter."""
    dense = {"kind": "dense", "ff": z["ff"]}
    moe = {"kind": "moe", "expert": {"ff": z["ff"] // 16}, "shared": {"ff": z["ff"] // 4},
           "router": {"experts": 32, "identity": 1, "top": 4, "scale": 2.5}}
    att = {"heads": z["heads"], "kv_heads": z["heads"] // 4, "dim": 64, "vdim": 64, "conv": 4, "scale": 0.125,
           "mask": {"size": window, "keep_first": keep_first}}
    dlt = {"heads": z["heads"], "kv_heads": z["heads"] // 4, "dim": 64, "vdim": 64, "conv": 4}
    kinds = [("attention", att, dense), ("attention", att, moe if experts else dense), ("delta", dlt, dense)]
    return {"architecture": "Solulix", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
            "layers": [{"type": kinds[i % 3][0], "mixer": kinds[i % 3][1], "mlp": kinds[i % 3][2]} for i in range(z["layers"])],
            "max_position_embeddings": CONTEXT_LEN}


def nonetar_config(z, window=1024, streams=4):
    """Six layers at the comparison's sizes: two layers of windowed attention (heads of 128 for the scores and 64 for
    the values, a quarter as many key/value heads, a window of 1024 tokens, capped scores) beside a gated diagonal
    recurrence as wide as the model (blocks of 64 channels, four taps), then one state-space-duality layer (twice the
    model's width in heads of 64 with a state of 128 rows, eight groups, four taps); four residual streams; dense
    feed-forwards of the same width as the other design's."""
    W, H = z["width"], z["heads"]
    mlp = {"kind": "dense", "ff": z["ff"]}
    par = {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": H, "kv_heads": H // 4, "dim": 128, "vdim": 64, "scale": 128 ** -0.5, "softcap": 30.0,
                 "mask": {"size": window}},
        "right": {"width": W, "blocks": W // 64, "conv": 4}, "left_scale": 1.0, "right_scale": 1.0}}
    ssd = {"type": "mamba2", "mlp": mlp, "mixer": {"heads": 2 * W // 64, "vdim": 64, "state": 128, "groups": 8,
                                                   "norm_groups": 8, "conv": 4}}
    return {"architecture": "Nonetar", "vocab": z["vocab"], "width": W, "norm": {"eps": 1e-6}, "streams": streams,
            "logit_scale": 1.0, "layers": [[par, par, ssd][i % 3] for i in range(z["layers"])],
            "max_position_embeddings": CONTEXT_LEN}


def tevanex_config(z, chunk=1024):
    """Six layers at the comparison's sizes: a matrix memory (heads of 64 x 64, the state of Solulix's delta rule), an
    attention with heads of 64 (a quarter as many key/value heads, every channel turning, a sink per head) and one with
    half as many heads of 128 (half of each head turning with stretched frequencies, capped scores, an output gate), both
    over blocks of 1024 positions; on every layer 32 experts of a thirty-second of the dense width of which a token uses
    four, and a shared expert of a quarter."""
    H = z["heads"]
    moe = {"kind": "moe", "expert": {"ff": z["ff"] // 32, "limit": 7.0}, "router": {"experts": 32, "top": 4},
           "shared": {"ff": z["ff"] // 4, "limit": 7.0}}
    mem = {"heads": H, "dim": 64, "vdim": 64, "gate_cap": 15.0}
    att = {"heads": H, "kv_heads": H // 4, "dim": 64, "vdim": 64, "scale": 0.125, "mask": {"size": chunk},
           "rot": {"base": 10000.0, "dims": 64}}
    att2 = {"heads": H // 2, "kv_heads": H // 8, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 30.0,
            "mask": {"size": chunk}, "rot": {"base": 10000.0, "dims": 64,
                                             "scaling": {"factor": 4.0, "original": 2048, "fast": 32.0, "slow": 1.0}}}
    kinds = [("mlstm", mem), ("attention", att), ("attention_2", att2)]
    return {"architecture": "Tevanex", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
            "embedding": {"scale": 1.0}, "residual_mult": 0.5, "logit_scale": 1.0, "logit_softcap": 30.0,
            "layers": [{"type": kinds[i % 3][0], "mixer": kinds[i % 3][1], "mlp": moe} for i in range(z["layers"])],
            "max_position_embeddings": CONTEXT_LEN}


def zatusun_config(z, chunk=1024):
    """Six layers at the comparison's sizes: a linear attention with a decay per channel (heads of 64 x 64, the state of
    Tevanex's matrix memory), a differential attention (half as many heads, two maps of 64 each over values of 128, a
    quarter as many key/value heads: the projections of Tevanex's attention; every channel turning, blocks of 1024
    positions) and a latent attention of Rezusun's sizes with an output gate; on every layer 32 experts of which a token
    uses four, together as wide as Tevanex's experts with their shared one; the last three layers are a run that goes
    through once."""
    H = z["heads"]
    moe = {"kind": "moe", "expert": {"ff": z["ff"] // 32 + z["ff"] // 128, "limit": 7.0}, "router": {"experts": 32, "top": 4}}
    lin = {"heads": H, "dim": 64, "vdim": 64}
    att = {"heads": H // 2, "kv_heads": H // 8, "dim": 64, "vdim": 128, "scale": 0.125, "diff": 0.5, "mask": {"size": chunk},
           "rot": {"base": 500000.0, "dims": 64, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 2048}}}
    lat = {"heads": z["lat_heads"], "dim": z["lat_dim"], "rot_dim": z["lat_rot"], "vdim": z["lat_vdim"], "q_rank": z["q_rank"],
           "kv_rank": z["kv_rank"], "scale": (z["lat_dim"] + z["lat_rot"]) ** -0.5,
           "rot": {"base": 10000.0, "dims": z["lat_rot"], "scaling": {"factor": 4.0, "original": 2048, "fast": 32.0, "slow": 1.0}}}
    kinds = [("hgrn2", lin), ("attention", att), ("latent_attention", lat)]
    n = z["layers"]
    return {"architecture": "Zatusun", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
            "embedding": {"scale": 1.0}, "logit_softcap": 30.0, "max_positions": CONTEXT_LEN,
            "layers": [{"type": kinds[i % 3][0], "mixer": kinds[i % 3][1], "mlp": moe} for i in range(n)],
            "loop": {"start": n // 2, "stop": n, "times": 1}}


def lobuzen_config(z, window=1024):
    """Six layers at the comparison's sizes: a latent attention of Rezusun's sizes (no rotated part, a sink per head), one
    that attends to that layer's latents, and an attention with heads of 64 and a quarter as many key/value heads, all three
    over a window of 1024 tokens; a dense feed-forward of Llama's width on the first layer, on the others 32 experts in four
    groups of which two are kept, four experts a token, of the width of Zatusun's; behind every layer a vector of a
    sixteenth of the width from each token."""
    H, W = z["heads"], z["width"]
    dense = {"kind": "dense", "ff": z["ff"], "limit": 7.0}
    moe = {"kind": "moe", "expert": {"ff": z["ff"] // 32 + z["ff"] // 128},
           "router": {"experts": 32, "top": 4, "groups": {"count": 4, "keep": 2}}}
    lat = {"heads": z["lat_heads"], "dim": z["lat_dim"], "vdim": z["lat_vdim"], "kv_rank": z["kv_rank"],
           "scale": z["lat_dim"] ** -0.5, "mask": {"size": window}}
    att = {"heads": H, "kv_heads": H // 4, "dim": 64, "vdim": 64, "scale": 0.125, "mask": {"size": window}}
    layers = []
    for i in range(z["layers"]):
        kind = i % 3
        mixer = att if kind == 2 else (dict(lat, kv_from=i - 1) if kind == 1 else lat)
        layers.append({"type": "attention" if kind == 2 else "latent_attention", "mixer": mixer, "mlp": moe if i else dense})
    return {"architecture": "Lobuzen", "vocab": z["vocab"], "width": W, "norm": {"eps": 1e-6}, "token_side": {"dim": W // 16},
            "layers": layers, "max_position_embeddings": CONTEXT_LEN}


def llama_config_like(z):
    cfg = dict(LLAMA_1B)
    cfg.update(hidden_size=z["width"], intermediate_size=z["ff"], vocab_size=z["vocab"], num_hidden_layers=z["layers"],
               num_attention_heads=z["heads"], num_key_value_heads=z["heads"] // 4, head_dim=64,
               tie_word_embeddings=False, max_position_embeddings=CONTEXT_LEN)
    return cfg


_compare_windows = []      # wall-clock intervals of the timed repetitions, for the clock samples


def _time_steps(fn, reps, warmup):
    import torch
    times = []
    for k in range(warmup + reps):
        if k == warmup:
            t_first = time.perf_counter()
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        start.record()
        fn(k)
        stop.record()
        torch.cuda.synchronize()
        if k >= warmup:
            times.append(start.elapsed_time(stop))
    _compare_windows.append((t_first, time.perf_counter()))
    return statistics.median(times)


def measure_design(config_dict, decode_batch=8, decode_batch_ops=64):
    """Prefill of one 2048-token portion and decode steps (from CUDA graphs) of a random model through the
    step function; then one launched step of each kind with an event behind every operator."""
    import numpy as np
    import torch
    from kv_cache_optimization_for_llm_b200 import EngineConfig, ops
    from kv_cache_optimization_for_llm_b200.engine.batch import StepEntry
    from kv_cache_optimization_for_llm_b200.engine.runner import ModelRunner
    seats = decode_batch_ops
    r = ModelRunner(None, EngineConfig(dtype="bfloat16", page_size=PAGE_SIZE, max_num_seqs=seats,
                                       num_pages=seats * (PROMPT_LEN + 64) // PAGE_SIZE + PREFILL_TOKENS // PAGE_SIZE,
                                       max_num_batched_tokens=PREFILL_TOKENS, max_model_len=CONTEXT_LEN),
                    random_init={"config": config_dict, "seed": 0, "std": 0.02})
    rng = np.random.default_rng(0)
    toks = rng.integers(0, r.vocab_size, PREFILL_TOKENS).tolist()

    def prefill(k):
        r.step([StepEntry(1000 + k, toks, 0, [PREFILL_TOKENS - 1])])
        r.release(1000 + k)
    out = {"weight_bytes": r.weight_bytes}
    ms = _time_steps(prefill, 5, 2)
    out["prefill_2048"] = {"ms": round(ms, 3), "tok_per_s": round(PREFILL_TOKENS / ms * 1e3)}
    with ops.timed_operators() as t:
        prefill(99)
    out["prefill_2048"]["operators"] = {k: [n, round(v, 3)] for k, (n, v) in sorted(t.times.items())}
    r.check_status()
    for batch, timed_ops in ((decode_batch, False), (decode_batch_ops, True)):
        prompts = [rng.integers(0, r.vocab_size, PROMPT_LEN + 48).tolist() for _ in range(batch)]
        for i in range(0, batch, 4):
            r.step([StepEntry(j, prompts[j][:PROMPT_LEN], 0, []) for j in range(i, min(batch, i + 4))])
        pos = [PROMPT_LEN]

        def decode(k):
            r.step([StepEntry(j, [prompts[j][pos[0]]], pos[0], [0]) for j in range(batch)])
            pos[0] += 1
        ms = _time_steps(decode, 24, 4)
        out[f"decode_b{batch}"] = {"ms_per_step": round(ms, 4), "tok_per_s": round(batch / ms * 1e3), "context": PROMPT_LEN}
        if timed_ops:
            buckets, r.graph_buckets = r.graph_buckets, []      # one step launched kernel by kernel
            decode(0)
            with ops.timed_operators() as t:
                decode(1)
            r.graph_buckets = buckets
            out[f"decode_b{batch}"]["operators_launched"] = {k: [n, round(v, 4)] for k, (n, v) in sorted(t.times.items())}
        for j in range(batch):
            r.release(j)
    r.check_status()
    del r
    torch.cuda.empty_cache()
    return out


def run_compare_solulix(size):
    """The Solulix design beside Llama at equal width, depth, feed-forward and vocabulary."""
    z = COMPARE_SIZES[size]
    pk = peaks()
    sampler = ClockSampler()
    sampler.start()
    w0 = time.perf_counter()
    log(f"{size}: Llama")
    llama = measure_design(llama_config_like(z))
    log(f"{size}: Solulix")
    window, keep = 1024, 64
    sol = measure_design(solulix_config(z, window, keep))
    w1 = time.perf_counter()
    sampler.stop()
    T, R, ctx = PREFILL_TOKENS, 64, PROMPT_LEN
    pairs = T * (T + 1) // 2
    # (query, key) pairs that the window and the kept first tokens leave of a T-token prompt
    seen = sum(min(i + 1, window) + max(0, min(keep, i + 1 - window)) for i in range(T))
    H, G, W = z["heads"], z["heads"] // 4, z["width"]
    channels = (H + 2 * G) * 64
    n_cols = 32 * (z["ff"] // 16) + z["ff"] // 4

    def per_launch(d, phase, key, *names):
        for name in names:
            n, ms = d[phase][key].get(name, (0, 0.0))
            if n:
                return ms / n
        return None

    def frac(work, ms, peak_per_s):
        return None if not ms else round(work / (ms * 1e-3) / peak_per_s, 4)
    tensor, hbm, fma = pk["bf16_tflops"] * 1e12, pk["hbm_gbs"] * 1e9, FP32_FMA_TFLOPS_NOMINAL * 1e12
    kernels = {
        "llama flash_attention, 2048 tokens (of the measured bf16 peak)": frac(
            pairs * 4 * H * 64, per_launch(llama, "prefill_2048", "operators", "paged_flash_attention"), tensor),
        "solulix attention, 2048 tokens (of the measured bf16 peak)": frac(
            seen * 4 * H * 64, per_launch(sol, "prefill_2048", "operators", "flash_attention_rows", "window_attention"), tensor),
        "llama decode_attention_mma, batch 64 (of the measured copy peak)": frac(
            R * ctx * 2 * G * 64 * 2, per_launch(llama, "decode_b64", "operators_launched", "decode_attention_mma"), hbm),
        "solulix window_attention, batch 64 (of the measured copy peak)": frac(
            R * min(ctx, window + keep) * 2 * G * 64 * 2, per_launch(sol, "decode_b64", "operators_launched", "window_attention"), hbm),
        "llama rope_kv_write, 2048 tokens (of the measured copy peak)": frac(
            T * (2 * channels + 2 * G * 64) * 2, per_launch(llama, "prefill_2048", "operators", "rope_kv_write"), hbm),
        # the convolution also writes the keys and values into their pages
        "solulix conv_silu, 2048 tokens (of the measured copy peak)": frac(
            T * 2 * channels * 2, per_launch(sol, "prefill_2048", "operators", "conv_silu"), hbm),
        "solulix delta_scan, 2048 tokens (of the nominal fp32 FMA peak)": frac(
            T * H * 64 * 64 * 10, per_launch(sol, "prefill_2048", "operators", "delta_scan"), fma),
        "solulix delta_scan, batch 64 (of the measured copy peak)": frac(
            2 * R * H * 64 * 64 * 4, per_launch(sol, "decode_b64", "operators_launched", "delta_scan"), hbm),
        "llama add_rmsnorm, 2048 tokens (of the measured copy peak)": frac(
            T * W * 12, per_launch(llama, "prefill_2048", "operators", "add_rmsnorm"), hbm),
        "solulix join_norm, 2048 tokens (of the measured copy peak)": frac(
            T * W * 14, per_launch(sol, "prefill_2048", "operators", "join_norm"), hbm),
        "solulix expert_act, 2048 tokens (of the measured copy peak)": frac(
            T * n_cols * 4, per_launch(sol, "prefill_2048", "operators", "expert_act"), hbm),
        "solulix route, 2048 tokens (of the nominal fp32 FMA peak)": frac(
            T * 33 * W * 2, per_launch(sol, "prefill_2048", "operators", "route"), fma),
    }
    return {"compare": size, "design": "solulix", "sizes": z, "window": window, "keep_first": keep, "dtype": "bf16",
            "data": "synthetic", "peaks": pk, "llama": llama, "solulix": sol, "kernel_roofline_fractions": kernels,
            "clocks": sampler.summary(list(_compare_windows) or [(w0, w1)])}


def run_compare_nonetar(size):
    """The Nonetar design beside Solulix (the closest design on the engine: windowed attention over [key | value]
    rows, short convolutions, a recurrence in state slots) at equal width, depth, dense feed-forward and vocabulary."""
    z = COMPARE_SIZES[size]
    pk = peaks()
    sampler = ClockSampler()
    sampler.start()
    w0 = time.perf_counter()
    window, keep, S = 1024, 64, 4
    log(f"{size}: Solulix (dense feed-forwards)")
    sol = measure_design(solulix_config(z, window, keep, experts=False))
    log(f"{size}: Nonetar")
    non = measure_design(nonetar_config(z, window, S))
    w1 = time.perf_counter()
    sampler.stop()
    T, R, ctx = PREFILL_TOKENS, 64, PROMPT_LEN
    seen_sol = sum(min(i + 1, window) + max(0, min(keep, i + 1 - window)) for i in range(T))
    seen = sum(min(i + 1, window) for i in range(T))
    H, G, W = z["heads"], z["heads"] // 4, z["width"]
    dk, dv = 128, 64
    sol_channels = (H + 2 * G) * 64
    C, Hs, N, Dv = W, 2 * W // 64, 128, 64
    inner, ssd_channels = Hs * Dv, Hs * Dv + 2 * 8 * N

    def per_launch(d, phase, key, *names):
        for name in names:
            n, ms = d[phase][key].get(name, (0, 0.0))
            if n:
                return ms / n
        return None

    def frac(work, ms, peak_per_s):
        return None if not ms else round(work / (ms * 1e-3) / peak_per_s, 4)
    tensor, hbm, fma = pk["bf16_tflops"] * 1e12, pk["hbm_gbs"] * 1e9, FP32_FMA_TFLOPS_NOMINAL * 1e12
    pre, dec = ("prefill_2048", "operators"), ("decode_b64", "operators_launched")
    kernels = {
        "solulix attention, 2048 tokens (of the measured bf16 peak)": frac(
            seen_sol * 4 * H * 64, per_launch(sol, *pre, "flash_attention_rows", "window_attention"), tensor),
        "nonetar window_attention, 2048 tokens (of the measured bf16 peak)": frac(
            seen * 2 * H * (dk + dv), per_launch(non, *pre, "window_flash_attention", "window_attention"), tensor),
        "solulix window_attention, batch 64 (of the measured copy peak)": frac(
            R * min(ctx, window + keep) * 2 * G * 64 * 2, per_launch(sol, *dec, "window_attention"), hbm),
        "nonetar window_attention, batch 64 (of the measured copy peak)": frac(
            R * min(ctx, window) * G * (dk + dv) * 2, per_launch(non, *dec, "window_attention"), hbm),
        # both also write the keys and values into their pages
        "solulix conv_silu, 2048 tokens (of the measured copy peak)": frac(
            T * 2 * sol_channels * 2, per_launch(sol, *pre, "conv_silu"), hbm),
        "nonetar conv_silu, 2048 tokens (of the measured copy peak)": frac(
            T * 2 * ((2 * C + ssd_channels) / 3) * 2, per_launch(non, *pre, "conv_silu"), hbm),
        "nonetar qk_norm_append, 2048 tokens (of the measured copy peak)": frac(
            T * ((H + G) * dk + G * dv + H * dk + G * (dk + dv)) * 2, per_launch(non, *pre, "qk_norm_append"), hbm),
        "solulix delta_scan, 2048 tokens (of the nominal fp32 FMA peak)": frac(
            T * H * 64 * 64 * 10, per_launch(sol, *pre, "delta_scan"), fma),
        "nonetar ssd_scan, 2048 tokens (of the nominal fp32 FMA peak)": frac(
            T * Hs * N * Dv * 5, per_launch(non, *pre, "ssd_scan"), fma),
        "solulix delta_scan, batch 64 (of the measured copy peak)": frac(
            2 * R * H * 64 * 64 * 4, per_launch(sol, *dec, "delta_scan"), hbm),
        "nonetar ssd_scan, batch 64 (of the measured copy peak)": frac(
            2 * R * Hs * N * Dv * 4, per_launch(non, *dec, "ssd_scan"), hbm),
        "nonetar coeffs_from_sums, 2048 tokens (of the measured copy peak)": frac(
            T * C * 18, per_launch(non, *pre, "coeffs_from_sums"), hbm),
        "nonetar diag_scan, 2048 tokens (of the measured copy peak)": frac(
            T * C * 12, per_launch(non, *pre, "diag_scan"), hbm),
        "nonetar diag_scan, batch 64 (of the measured copy peak)": frac(
            R * C * 20, per_launch(non, *dec, "diag_scan"), hbm),
        "nonetar gated_group_norm, 2048 tokens (of the measured copy peak)": frac(
            T * inner * 8, per_launch(non, *pre, "gated_group_norm"), hbm),
        "solulix join_norm, 2048 tokens (of the measured copy peak)": frac(
            T * W * 14, per_launch(sol, *pre, "join_norm"), hbm),
        # reads and writes every stream in float32, reads the sublayer's output, writes the next one's input
        "nonetar hyper_norm, 2048 tokens (of the measured copy peak)": frac(
            T * W * (8 * S + 6), per_launch(non, *pre, "hyper_norm"), hbm),
        "nonetar token_shift, 2048 tokens (of the measured copy peak)": frac(
            T * W * 6, per_launch(non, *pre, "token_shift"), hbm),
        "nonetar xielu, 2048 tokens (of the measured copy peak)": frac(
            T * z["ff"] * 4, per_launch(non, *pre, "xielu"), hbm),
    }
    return {"compare": size, "design": "nonetar", "beside": "solulix", "sizes": z, "window": window, "streams": S,
            "dtype": "bf16", "data": "synthetic", "peaks": pk, "solulix": sol, "nonetar": non,
            "kernel_roofline_fractions": kernels, "clocks": sampler.summary(list(_compare_windows) or [(w0, w1)])}


def run_compare_tevanex(size):
    """The Tevanex design beside Solulix (the closest design on the engine: attention over [key | value] rows in a
    windowed page group, a matrix state per head in state slots, routed experts computed for every token) at equal
    width, depth and vocabulary."""
    z = COMPARE_SIZES[size]
    pk = peaks()
    sampler = ClockSampler()
    sampler.start()
    w0 = time.perf_counter()
    window, keep, chunk = 1024, 64, 1024
    log(f"{size}: Solulix")
    sol = measure_design(solulix_config(z, window, keep))
    log(f"{size}: Tevanex")
    tev = measure_design(tevanex_config(z, chunk))
    w1 = time.perf_counter()
    sampler.stop()
    T, R, ctx = PREFILL_TOKENS, 64, PROMPT_LEN
    seen_sol = sum(min(i + 1, window) + max(0, min(keep, i + 1 - window)) for i in range(T))
    seen = sum(i % chunk + 1 for i in range(T))
    H, G, W = z["heads"], z["heads"] // 4, z["width"]
    sol_channels = (H + 2 * G) * 64
    sol_cols = 32 * (z["ff"] // 16) + z["ff"] // 4
    cols = 32 * (z["ff"] // 32) + z["ff"] // 4
    # per token: the product's q, k, v read, the queries written, the rows [k | v] written (the two attentions' mean)
    qkv_elems = ((H + 2 * G) * 64 + (H // 2 + 2 * (H // 8)) * 128) / 2

    def per_launch(d, phase, key, *names):
        for name in names:
            n, ms = d[phase][key].get(name, (0, 0.0))
            if n:
                return ms / n
        return None

    def frac(work, ms, peak_per_s):
        return None if not ms else round(work / (ms * 1e-3) / peak_per_s, 4)
    tensor, hbm, fma = pk["bf16_tflops"] * 1e12, pk["hbm_gbs"] * 1e9, FP32_FMA_TFLOPS_NOMINAL * 1e12
    pre, dec = ("prefill_2048", "operators"), ("decode_b64", "operators_launched")
    kernels = {
        "solulix attention, 2048 tokens (of the measured bf16 peak)": frac(
            seen_sol * 4 * H * 64, per_launch(sol, *pre, "flash_attention_rows", "window_attention"), tensor),
        # both attentions do 2 (dk + dv) heads = 256 H FLOP per seen pair
        # the tcgen05 kernel where its 128-row tiles fill the GPU, else the mma.sync kernel
        "tevanex attention, 2048 tokens (of the measured bf16 peak)": frac(
            seen * 4 * H * 64, per_launch(tev, *pre, "flash_attention_rows", "window_flash_attention", "window_attention"), tensor),
        "solulix window_attention, batch 64 (of the measured copy peak)": frac(
            R * min(ctx, window + keep) * 2 * G * 64 * 2, per_launch(sol, *dec, "window_attention"), hbm),
        "tevanex window_attention, batch 64 (of the measured copy peak)": frac(
            R * min(ctx, chunk) * 2 * G * 64 * 2, per_launch(tev, *dec, "window_attention"), hbm),
        # both also write the keys and values into their pages
        "solulix conv_silu, 2048 tokens (of the measured copy peak)": frac(
            T * 2 * sol_channels * 2, per_launch(sol, *pre, "conv_silu"), hbm),
        "tevanex qk_rot_append, 2048 tokens (of the measured copy peak)": frac(
            T * 2 * qkv_elems * 2, per_launch(tev, *pre, "qk_rot_append"), hbm),
        "solulix delta_scan, 2048 tokens (of the nominal fp32 FMA peak)": frac(
            T * H * 64 * 64 * 10, per_launch(sol, *pre, "delta_scan"), fma),
        # per element of the memory and token: keep and add (2 FLOP), read out (2); the vector n is 1/64 more
        "tevanex mlstm_scan, 2048 tokens (of the nominal fp32 FMA peak)": frac(
            T * H * 64 * 65 * 4, per_launch(tev, *pre, "mlstm_scan"), fma),
        "solulix delta_scan, batch 64 (of the measured copy peak)": frac(
            2 * R * H * 64 * 64 * 4, per_launch(sol, *dec, "delta_scan"), hbm),
        "tevanex mlstm_scan, batch 64 (of the measured copy peak)": frac(
            2 * R * H * 64 * 65 * 4, per_launch(tev, *dec, "mlstm_scan"), hbm),
        "tevanex head_norm_gate, 2048 tokens (of the measured copy peak)": frac(
            T * H * 64 * 8, per_launch(tev, *pre, "head_norm_gate"), hbm),
        "solulix join_norm, 2048 tokens (of the measured copy peak)": frac(
            T * W * 14, per_launch(sol, *pre, "join_norm"), hbm),
        # the branch output read, the float32 stream read and written, the next sublayer's input written
        "tevanex add_norm, 2048 tokens (of the measured copy peak)": frac(
            T * W * 12, per_launch(tev, *pre, "add_norm"), hbm),
        "solulix expert_act, 2048 tokens (of the measured copy peak)": frac(
            T * sol_cols * 4, per_launch(sol, *pre, "expert_act"), hbm),
        # two products read, one activation written
        "tevanex limited_act, 2048 tokens (of the measured copy peak)": frac(
            T * cols * 6, per_launch(tev, *pre, "limited_act"), hbm),
        "solulix route, 2048 tokens (of the nominal fp32 FMA peak)": frac(
            T * 33 * W * 2, per_launch(sol, *pre, "route"), fma),
        # the logits come from a matrix product; the kernel reads them and writes the weights
        "tevanex route, 2048 tokens (of the measured copy peak)": frac(
            T * (33 + 32) * 4, per_launch(tev, *pre, "route"), hbm),
    }
    return {"compare": size, "design": "tevanex", "beside": "solulix", "sizes": z, "window": window, "chunk": chunk,
            "dtype": "bf16", "data": "synthetic", "peaks": pk, "solulix": sol, "tevanex": tev,
            "kernel_roofline_fractions": kernels, "clocks": sampler.summary(list(_compare_windows) or [(w0, w1)])}


def run_compare_zatusun(size):
    """The Zatusun design beside Tevanex (the closest design on the engine: attention over blocks of positions in a
    windowed page group, a matrix state per head in state slots, limited experts computed for every token) at equal
    width, depth and vocabulary; the latent attention's kernels beside Rezusun's at equal sizes."""
    z = COMPARE_SIZES[size]
    pk = peaks()
    sampler = ClockSampler()
    sampler.start()
    w0 = time.perf_counter()
    chunk = 1024
    log(f"{size}: Tevanex")
    tev = measure_design(tevanex_config(z, chunk))
    log(f"{size}: Rezusun")
    rez = measure_design(rezusun_config(z))
    log(f"{size}: Zatusun")
    zat = measure_design(zatusun_config(z, chunk))
    w1 = time.perf_counter()
    sampler.stop()
    T, R, ctx = PREFILL_TOKENS, 64, PROMPT_LEN
    pairs = T * (T + 1) // 2
    seen = sum(i % chunk + 1 for i in range(T))
    H, G, W = z["heads"], z["heads"] // 4, z["width"]
    dc = z["kv_rank"] + z["lat_rot"]
    cols = 32 * (z["ff"] // 32) + z["ff"] // 4
    # per token: the product's q, k, v read, the queries written, the rows written (Tevanex: the two attentions' mean)
    tev_qkv = ((H + 2 * G) * 64 + (H // 2 + 2 * (H // 8)) * 128) / 2
    zat_qkv = (H + 2 * G) * 64

    def per_launch(d, phase, key, *names):
        for name in names:
            n, ms = d[phase][key].get(name, (0, 0.0))
            if n:
                return ms / n
        return None

    def frac(work, ms, peak_per_s):
        return None if not ms else round(work / (ms * 1e-3) / peak_per_s, 4)
    tensor, hbm, fma = pk["bf16_tflops"] * 1e12, pk["hbm_gbs"] * 1e9, FP32_FMA_TFLOPS_NOMINAL * 1e12
    pre, dec = ("prefill_2048", "operators"), ("decode_b64", "operators_launched")
    lat_names = ("latent_attention_tc", "latent_attention")
    kernels = {
        "tevanex attention, 2048 tokens (of the measured bf16 peak)": frac(
            seen * 4 * H * 64, per_launch(tev, *pre, "flash_attention_rows", "window_flash_attention", "window_attention"), tensor),
        # two maps a head: 2 (dim + vdim) FLOP each per seen pair
        "zatusun attention, 2048 tokens (of the measured bf16 peak)": frac(
            seen * 2 * (64 + 128) * 2 * (H // 2), per_launch(zat, *pre, "window_flash_attention", "window_attention"), tensor),
        "tevanex window_attention, batch 64 (of the measured copy peak)": frac(
            R * min(ctx, chunk) * 2 * G * 64 * 2, per_launch(tev, *dec, "window_attention"), hbm),
        "zatusun window_attention, batch 64 (of the measured copy peak)": frac(
            R * min(ctx, chunk) * (H // 8) * 256 * 2, per_launch(zat, *dec, "window_attention"), hbm),
        "tevanex qk_rot_append, 2048 tokens (of the measured copy peak)": frac(
            T * 2 * tev_qkv * 2, per_launch(tev, *pre, "qk_rot_append"), hbm),
        "zatusun qk_rot_append, 2048 tokens (of the measured copy peak)": frac(
            T * 2 * zat_qkv * 2, per_launch(zat, *pre, "qk_rot_append"), hbm),
        # per element of the memory and token: keep and add (2 FLOP), read out (2)
        "tevanex mlstm_scan, 2048 tokens (of the nominal fp32 FMA peak)": frac(
            T * H * 64 * 65 * 4, per_launch(tev, *pre, "mlstm_scan"), fma),
        "zatusun linear_scan, 2048 tokens (of the nominal fp32 FMA peak)": frac(
            T * H * 64 * 64 * 4, per_launch(zat, *pre, "linear_scan"), fma),
        "tevanex mlstm_scan, batch 64 (of the measured copy peak)": frac(
            2 * R * H * 64 * 65 * 4, per_launch(tev, *dec, "mlstm_scan"), hbm),
        "zatusun linear_scan, batch 64 (of the measured copy peak)": frac(
            2 * R * H * 64 * 64 * 4, per_launch(zat, *dec, "linear_scan"), hbm),
        "rezusun latent_attention, 2048 tokens (of the measured bf16 peak)": frac(
            pairs * z["lat_heads"] * 2 * (dc + z["kv_rank"]), per_launch(rez, *pre, *lat_names), tensor),
        "zatusun latent_attention, 2048 tokens (of the measured bf16 peak)": frac(
            pairs * z["lat_heads"] * 2 * (dc + z["kv_rank"]), per_launch(zat, *pre, *lat_names), tensor),
        "rezusun latent_attention, batch 64 (of the measured copy peak)": frac(
            R * ctx * dc * 2, per_launch(rez, *dec, *lat_names), hbm),
        "zatusun latent_attention, batch 64 (of the measured copy peak)": frac(
            R * ctx * dc * 2, per_launch(zat, *dec, *lat_names), hbm),
        "rezusun latent_prep, 2048 tokens (of the measured copy peak)": frac(
            T * 2 * (z["q_rank"] + dc) * 2, per_launch(rez, *pre, "latent_prep"), hbm),
        "zatusun latent_prep, 2048 tokens (of the measured copy peak)": frac(
            T * 2 * (z["q_rank"] + dc) * 2, per_launch(zat, *pre, "latent_prep"), hbm),
        "tevanex add_norm, 2048 tokens (of the measured copy peak)": frac(
            T * W * 12, per_launch(tev, *pre, "add_norm"), hbm),
        "zatusun add_rmsnorm, 2048 tokens (of the measured copy peak)": frac(
            T * W * 12, per_launch(zat, *pre, "add_rmsnorm"), hbm),
        # the start of a pass: the product's rows and the embedding's share read, the stream and the normed rows written
        "zatusun join_norm, 2048 tokens (of the measured copy peak)": frac(
            T * W * 14, per_launch(zat, *pre, "join_norm"), hbm),
        "tevanex limited_act, 2048 tokens (of the measured copy peak)": frac(
            T * cols * 6, per_launch(tev, *pre, "limited_act"), hbm),
        "zatusun limited_act, 2048 tokens (of the measured copy peak)": frac(
            T * cols * 6, per_launch(zat, *pre, "limited_act"), hbm),
        "tevanex route, 2048 tokens (of the measured copy peak)": frac(T * (33 + 32) * 4, per_launch(tev, *pre, "route"), hbm),
        "zatusun route, 2048 tokens (of the measured copy peak)": frac(T * (32 + 32) * 4, per_launch(zat, *pre, "route"), hbm),
    }
    return {"compare": size, "design": "zatusun", "beside": "tevanex, rezusun", "sizes": z, "chunk": chunk, "dtype": "bf16",
            "data": "synthetic", "peaks": pk, "tevanex": tev, "rezusun": rez, "zatusun": zat,
            "kernel_roofline_fractions": kernels, "clocks": sampler.summary(list(_compare_windows) or [(w0, w1)])}


def run_compare_lobuzen(size):
    """The Lobuzen design beside the two closest on the engine at equal width, depth and vocabulary: Zatusun (latent
    attention, experts without a shared one) and Tevanex (norms behind the sublayers only, attention with heads of 64 over
    [key | value] rows in a windowed page group)."""
    z = COMPARE_SIZES[size]
    pk = peaks()
    sampler = ClockSampler()
    sampler.start()
    w0 = time.perf_counter()
    window = 1024
    log(f"{size}: Tevanex")
    tev = measure_design(tevanex_config(z, window))
    log(f"{size}: Zatusun")
    zat = measure_design(zatusun_config(z, window))
    log(f"{size}: Lobuzen")
    lob = measure_design(lobuzen_config(z, window))
    w1 = time.perf_counter()
    sampler.stop()
    T, R, ctx = PREFILL_TOKENS, 64, PROMPT_LEN
    H, G, W, n = z["heads"], z["heads"] // 4, z["width"], z["layers"]
    pairs = T * (T + 1) // 2
    seen = sum(min(i + 1, window) for i in range(T))
    in_block = sum(i % window + 1 for i in range(T))
    dc, kr, side = z["kv_rank"] + z["lat_rot"], z["kv_rank"], z["width"] // 16
    tev_cols = 32 * (z["ff"] // 32) + z["ff"] // 4
    moe_cols = 32 * (z["ff"] // 32 + z["ff"] // 128)
    lob_cols = (z["ff"] + (n - 1) * moe_cols) / n
    tev_qkv = ((H + 2 * G) * 64 + (H // 2 + 2 * (H // 8)) * 128) / 2

    def per_launch(d, phase, key, *names):
        for name in names:
            calls, ms = d[phase][key].get(name, (0, 0.0))
            if calls:
                return ms / calls
        return None

    def frac(work, ms, peak_per_s):
        return None if not ms else round(work / (ms * 1e-3) / peak_per_s, 4)
    tensor, hbm = pk["bf16_tflops"] * 1e12, pk["hbm_gbs"] * 1e9
    pre, dec = ("prefill_2048", "operators"), ("decode_b64", "operators_launched")
    lat_names = ("latent_attention_tc", "latent_attention")
    att_names = ("flash_attention_rows", "window_flash_attention", "window_attention")
    # a long run of Lobuzen's latent layers attends to keys and values that were made for it, on the kernels of its other
    # attention: all layers together
    lob_att_ms = sum(lob["prefill_2048"]["operators"].get(k, (0, 0.0))[1] for k in att_names)
    lat_up = 2 * z["lat_heads"] * (z["lat_dim"] + z["lat_vdim"]) * kr * T
    kernels = {
        "zatusun latent_attention, 2048 tokens (of the measured bf16 peak)": frac(
            pairs * z["lat_heads"] * 2 * (dc + kr), per_launch(zat, *pre, *lat_names), tensor),
        "lobuzen attention of all layers, 2048 tokens (of the measured bf16 peak)": frac(
            seen * 2 * ((n - n // 3) * z["lat_heads"] * (z["lat_dim"] + z["lat_vdim"]) + n // 3 * H * 128), lob_att_ms, tensor),
        "lobuzen latent_rows, 2048 tokens (of the measured copy peak)": frac(T * kr * 4, per_launch(lob, *pre, "latent_rows"), hbm),
        "lobuzen keys and values of a latent, 2048 tokens (of the measured bf16 peak)": frac(
            lat_up, per_launch(lob, *pre, "latent_up_library"), tensor),
        "zatusun latent_attention, batch 64 (of the measured copy peak)": frac(
            R * ctx * dc * 2, per_launch(zat, *dec, *lat_names), hbm),
        "lobuzen latent_attention, batch 64 (of the measured copy peak)": frac(
            R * min(ctx, window) * kr * 2, per_launch(lob, *dec, "latent_decode", *lat_names), hbm),
        "zatusun latent_prep, 2048 tokens (of the measured copy peak)": frac(
            T * 2 * (z["q_rank"] + dc) * 2, per_launch(zat, *pre, "latent_prep"), hbm),
        "lobuzen latent_prep, 2048 tokens (of the measured copy peak)": frac(
            T * 2 * kr * 2, per_launch(lob, *pre, "latent_prep"), hbm),
        "tevanex attention, 2048 tokens (of the measured bf16 peak)": frac(
            in_block * 4 * H * 64, per_launch(tev, *pre, *att_names), tensor),
        "tevanex window_attention, batch 64 (of the measured copy peak)": frac(
            R * min(ctx, window) * 2 * G * 64 * 2, per_launch(tev, *dec, "window_attention"), hbm),
        "lobuzen window_attention, batch 64 (of the measured copy peak)": frac(
            R * min(ctx, window) * 2 * G * 64 * 2, per_launch(lob, *dec, "window_attention"), hbm),
        "tevanex qk_rot_append, 2048 tokens (of the measured copy peak)": frac(
            T * 2 * tev_qkv * 2, per_launch(tev, *pre, "qk_rot_append"), hbm),
        "lobuzen qk_norm_append, 2048 tokens (of the measured copy peak)": frac(
            T * 2 * (H + 2 * G) * 64 * 2, per_launch(lob, *pre, "qk_norm_append"), hbm),
        "tevanex add_norm, 2048 tokens (of the measured copy peak)": frac(T * W * 12, per_launch(tev, *pre, "add_norm"), hbm),
        "lobuzen add_norm, 2048 tokens (of the measured copy peak)": frac(T * W * 12, per_launch(lob, *pre, "add_norm"), hbm),
        "tevanex limited_act, 2048 tokens (of the measured copy peak)": frac(
            T * tev_cols * 6, per_launch(tev, *pre, "limited_act"), hbm),
        "zatusun limited_act, 2048 tokens (of the measured copy peak)": frac(
            T * moe_cols * 6, per_launch(zat, *pre, "limited_act"), hbm),
        "lobuzen limited_act, 2048 tokens (of the measured copy peak)": frac(
            T * lob_cols * 6, per_launch(lob, *pre, "limited_act"), hbm),
        "zatusun route, 2048 tokens (of the measured copy peak)": frac(T * (32 + 32) * 4, per_launch(zat, *pre, "route"), hbm),
        "lobuzen route, 2048 tokens (of the measured copy peak)": frac(T * (32 + 32) * 4, per_launch(lob, *pre, "route"), hbm),
        # the gate products and the table's rows read, the gated rows written
        "lobuzen token_gate, 2048 tokens (of the measured copy peak)": frac(T * side * 6, per_launch(lob, *pre, "token_gate"), hbm),
        # both matrices, the pending branch output read, the stream read and written, its copy written
        "lobuzen token_input_step, batch 64 (of the measured copy peak)": frac(
            2 * W * side * 2 + R * W * 12, per_launch(lob, *dec, "token_input_step"), hbm),
    }
    return {"compare": size, "design": "lobuzen", "beside": "tevanex, zatusun", "sizes": z, "window": window, "dtype": "bf16",
            "data": "synthetic", "peaks": pk, "tevanex": tev, "zatusun": zat, "lobuzen": lob,
            "kernel_roofline_fractions": kernels, "clocks": sampler.summary(list(_compare_windows) or [(w0, w1)])}


def run_compare(size):
    """The Rezusun design beside Llama at equal width, depth, feed-forward and vocabulary."""
    z = COMPARE_SIZES[size]
    pk = peaks()
    sampler = ClockSampler()
    sampler.start()
    w0 = time.perf_counter()
    log(f"{size}: Llama")
    llama = measure_design(llama_config_like(z))
    log(f"{size}: Rezusun")
    rez = measure_design(rezusun_config(z))
    w1 = time.perf_counter()
    sampler.stop()
    T, R, ctx = PREFILL_TOKENS, 64, PROMPT_LEN
    pairs = T * (T + 1) // 2
    n_each = z["layers"] // 3
    H, Dk = z["heads"], 64
    dc = z["kv_rank"] + z["lat_rot"]

    def per_launch(d, phase, key, *names):
        """Milliseconds per call of the operator (the first of ``names`` that the step used)."""
        for name in names:
            n, ms = d[phase][key].get(name, (0, 0.0))
            if n:
                return ms / n
        return None

    def frac(work, ms, peak_per_s):
        return None if not ms else round(work / (ms * 1e-3) / peak_per_s, 4)
    tensor, hbm, fma = pk["bf16_tflops"] * 1e12, pk["hbm_gbs"] * 1e9, FP32_FMA_TFLOPS_NOMINAL * 1e12
    kernels = {
        # prefill: FLOPs of the kernel's own arithmetic over the time of one launch
        "llama flash_attention, 2048 tokens (of the measured bf16 peak)": frac(
            pairs * 4 * z["heads"] * 64, per_launch(llama, "prefill_2048", "operators", "paged_flash_attention"), tensor),
        "rezusun latent_attention, 2048 tokens (of the measured bf16 peak)": frac(
            pairs * z["lat_heads"] * 2 * (dc + z["kv_rank"]),
            per_launch(rez, "prefill_2048", "operators", "latent_attention_tc", "latent_attention"), tensor),
        "rezusun delta_scan, 2048 tokens (of the nominal fp32 FMA peak)": frac(
            T * H * Dk * 64 * 10, per_launch(rez, "prefill_2048", "operators", "delta_scan"), fma),
        # decode, 64 requests at 512 tokens: bytes that must move over the time of one launch
        "llama decode_attention_mma, batch 64 (of the measured copy peak)": frac(
            R * ctx * 2 * (z["heads"] // 4) * 64 * 2, per_launch(llama, "decode_b64", "operators_launched", "decode_attention_mma"), hbm),
        "rezusun latent_attention, batch 64 (of the measured copy peak)": frac(
            R * ctx * dc * 2, per_launch(rez, "decode_b64", "operators_launched", "latent_attention_tc", "latent_attention"), hbm),
        "rezusun delta_scan, batch 64 (of the measured copy peak)": frac(
            2 * R * H * 64 * Dk * 4, per_launch(rez, "decode_b64", "operators_launched", "delta_scan"), hbm),
        "llama add_rmsnorm, 2048 tokens (of the measured copy peak)": frac(
            T * z["width"] * 12, per_launch(llama, "prefill_2048", "operators", "add_rmsnorm"), hbm),
        "rezusun add_norm, 2048 tokens (of the measured copy peak)": frac(
            T * z["width"] * 12, per_launch(rez, "prefill_2048", "operators", "add_norm"), hbm),
    }
    return {"compare": size, "sizes": z, "dtype": "bf16", "data": "synthetic", "peaks": pk, "llama": llama, "rezusun": rez,
            "kernel_roofline_fractions": kernels, "layers_of_each_kind": n_each,
            "clocks": sampler.summary(list(_compare_windows) or [(w0, w1)])}


def main():
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=128)
    ap.add_argument("--warmup", type=int, default=16)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--layers", type=int, default=FULL_LAYERS, help="fewer layers than the model has (named in config)")
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--skip-points", action="store_true", help="skip batch 1 / 64 and the prefill measurement")
    ap.add_argument("--check", action="store_true",
                    help="also compare logits of a 2-layer model of these widths with the plain implementation under "
                         "tests/ on the timed paths (adds about a minute); the line gets a \"check\" key and the exit "
                         "code is 1 if the limit is broken")
    ap.add_argument("--workload", default="all", choices=["all", "none", *WORKLOADS],
                    help="the serving workloads measured beside the headline (3B continuous batching, 8B under a "
                         "pool that is too small); one name runs that workload alone and prints its own JSON line")
    ap.add_argument("--compare", default=None, choices=sorted(COMPARE_SIZES),
                    help="instead of the headline: prefill and decode of another design (--design) beside a Llama model of "
                         "equal width, depth, feed-forward and vocabulary (random weights), with the time of every "
                         "operator and roofline fractions of the designs' own kernels; prints its own JSON line")
    ap.add_argument("--design", default="rezusun", choices=["rezusun", "solulix", "nonetar", "tevanex", "zatusun", "lobuzen"],
                    help="with --compare: which design stands beside Llama (nonetar and tevanex: beside Solulix; zatusun: "
                         "beside Tevanex and Rezusun; lobuzen: beside Tevanex and Zatusun, the closest designs)")
    args = ap.parse_args()

    if args.compare:
        result = {"solulix": run_compare_solulix, "nonetar": run_compare_nonetar,
                  "tevanex": run_compare_tevanex, "zatusun": run_compare_zatusun,
                  "lobuzen": run_compare_lobuzen}.get(args.design, run_compare)(args.compare)
        print(json.dumps(result), flush=True)
        return 0
    if args.impl == "reference":
        # upstream's own engine, unmodified, driven through its standard input and output
        sys.path.insert(0, os.path.join(ROOT, "baseline"))
        import reference_arm
        return reference_arm.run(args, dict(LLAMA_1B), PROMPT_LEN, NEW_TOKENS, ClockSampler)
    if args.gpus != 1:
        print(f"bench.py measures one GPU only (this engine runs on one GPU); got --gpus {args.gpus}")
        return 2
    if args.steps < 1 or args.warmup < 3 or args.steps + args.warmup + 2 > NEW_TOKENS:
        print(f"need steps >= 1, warmup >= 3 and steps + warmup + 2 <= {NEW_TOKENS}")
        return 2

    import torch
    from kv_cache_optimization_for_llm_b200 import LLM

    if args.workload in WORKLOADS:
        print(json.dumps({"workload": args.workload, **run_workload(args.workload)}), flush=True)
        return 0
    cfg = dict(LLAMA_1B)
    cfg["num_hidden_layers"] = args.layers
    pk = peaks()
    nums = model_numbers(cfg, args.layers)
    max_batch = max(args.batch, 1 if args.skip_points else 64)
    log(f"building Llama-3.2-1B shape, {args.layers} layers, random bfloat16 weights")
    llm = LLM.from_random(cfg, seed=0, std=0.02, dtype="bfloat16", page_size=PAGE_SIZE,
                          num_pages=max_batch * (CONTEXT_LEN // PAGE_SIZE) // 4 + PREFILL_TOKENS // PAGE_SIZE,
                          max_num_seqs=max_batch, max_num_batched_tokens=PREFILL_TOKENS, max_model_len=CONTEXT_LEN)
    sampler = ClockSampler()
    sampler.start()
    windows = []

    log(f"decode, batch {args.batch}: device-timed")
    sec, mean_ctx, launches, win = run_decode(llm, args.batch, args.steps, args.warmup, False, seed=1)
    windows.append(win)
    value = args.batch * args.steps / sec
    ms_per_step = 1000.0 * sec / args.steps
    log(f"  {value:.0f} tok/s, {ms_per_step:.3f} ms/step, {launches} launches")
    log(f"decode, batch {args.batch}: end to end")
    sec_e, _, _, win = run_decode(llm, args.batch, args.steps, args.warmup, True, seed=1)
    windows.append(win)
    e2e = args.batch * args.steps / sec_e
    b_in = run_decode.h2d_bytes + 4 * 4 * args.batch   # batch arrays + sampler parameters
    log(f"  {e2e:.0f} tok/s")

    step_bytes = nums["weight_bytes"] + args.batch * mean_ctx * nums["kv_bytes_per_token"]
    achieved = step_bytes / (ms_per_step / 1000.0) / 1e9
    points, point_rooflines, prefill = {}, {}, None
    if not args.skip_points:
        for b in (1, 64):
            log(f"decode, batch {b}")
            s, ctx_b, _, win = run_decode(llm, b, args.steps, args.warmup, False, seed=2 + b)
            windows.append(win)
            points[f"decode_b{b}"] = round(b * args.steps / s, 1)
            bytes_b = nums["weight_bytes"] + b * ctx_b * nums["kv_bytes_per_token"]
            gbs = bytes_b / (s / args.steps) / 1e9
            point_rooflines[f"decode_b{b}"] = {"ms_per_step": round(1000.0 * s / args.steps, 4), "bytes": int(bytes_b),
                                               "achieved": round(gbs, 1), "frac": round(gbs / pk["hbm_gbs"], 4)}
            log(f"  {points[f'decode_b{b}']:.0f} tok/s, {gbs:.0f} GB/s = {gbs / pk['hbm_gbs']:.3f} of {pk['source']} HBM peak")
        log(f"prefill of {PREFILL_TOKENS} tokens")
        w0 = time.perf_counter()
        ms = run_prefill(llm, reps=5, warmup=3, seed=9)
        windows.append((w0, time.perf_counter()))
        fl = prefill_flops(cfg, args.layers, PREFILL_TOKENS)
        prefill = {"value": round(PREFILL_TOKENS / (ms / 1000.0), 1), "tokens": PREFILL_TOKENS, "ms": round(ms, 3),
                   "frac": round(fl / (ms / 1000.0) / (pk["bf16_tflops"] * 1e12), 4)}
        log(f"  {prefill['value']:.0f} tok/s, {ms:.2f} ms, {prefill['frac']:.3f} of {pk['source']} bf16 peak")
        log("time to the first token of a lone 128-token prompt")
        w0 = time.perf_counter()
        points["first_token_ms_prompt128"] = round(run_first_token(llm, 128, reps=7, warmup=3, seed=13), 3)
        windows.append((w0, time.perf_counter()))
        log(f"  {points['first_token_ms_prompt128']:.2f} ms")
    sampler.stop()
    clocks = sampler.summary(windows)
    b_out = 4 * args.batch + 4                                              # sampled ids + the status word
    graphs_on = bool(llm.engine.config.use_cuda_graphs)
    workloads = {}
    if args.workload == "all" and not args.skip_points:
        del llm
        import gc
        gc.collect()
        torch.cuda.empty_cache()
        for name in WORKLOADS:
            try:
                workloads[name] = run_workload(name)
            except Exception as e:       # the headline must not be lost to a side measurement
                workloads[name] = {"error": f"{type(e).__name__}: {e}"[:300]}
                log(f"{name} failed: {workloads[name]['error']}")

    line = {
        "metric": "decode tok/s (Llama-3.2-1B shape, bf16, batch 8, 512-token prompts)",
        "value": round(value, 1), "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
        "ms_per_step": round(ms_per_step, 4), "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic: uniform-random token ids, random-init weights N(0,0.02)",
        "impl": "ours",
        "config": {
            "model": "Llama-3.2-1B shape (LlamaForCausalLM)", "layers": args.layers, "layers_full_model": FULL_LAYERS,
            "hidden_size": cfg["hidden_size"], "intermediate_size": cfg["intermediate_size"],
            "num_attention_heads": cfg["num_attention_heads"], "num_key_value_heads": cfg["num_key_value_heads"],
            "head_dim": cfg["head_dim"], "vocab_size": cfg["vocab_size"], "tied_lm_head": True,
            "global_batch": args.batch, "prompt_len": PROMPT_LEN, "new_tokens": NEW_TOKENS,
            "context_len": CONTEXT_LEN, "page_size": PAGE_SIZE, "kv_dtype": "bf16", "parallelism": "none (1 GPU)",
            "l2": "inputs larger than L2: 2.47 GB of weights are streamed every step",
            "cuda_graphs": graphs_on,
        },
        "e2e": {"value": round(e2e, 1), "unit": "tokens/s", "h2d_bytes_per_step": int(b_in),
                "d2h_bytes_per_step": int(b_out)},
        "gpu_launches": int(launches),
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4), "peak_source": pk["source"], "bytes": int(step_bytes),
                     "points": point_rooflines},
        "clocks": clocks,
    }
    if prefill is not None:
        line["prefill"] = prefill
    if points:
        line["points"] = points
    if workloads:
        line["workloads"] = workloads
    if args.check:
        log("logits of a 2-layer model of these widths against the plain implementation")
        line["check"] = run_value_check(dict(LLAMA_1B))
        log(f"  {line['check']}")
    print(json.dumps(line), flush=True)
    return 0 if not args.check or line["check"]["ok"] else 1


if __name__ == "__main__":
    sys.exit(main())
