#!/usr/bin/env python3
"""Headline benchmark: decode throughput of the Qwen2.5-0.5B shape (random weights, bfloat16) at a
batch of 8 and a context of 4,096 tokens on ONE B200, with prefill of 2,048 tokens, the decode
roofline and batch 1 / 64 points on the same JSON line.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference] [--shape 0.5b|1.5b|7b]

A "step" is one decode step of the whole batch. ``value`` is decoded tokens per second over K steps
timed with CUDA events on the launching stream; ``e2e`` is the same through the Python entry point
(the scheduler with lookahead, as ``Model.generate`` and the serve command run it: host token ids in,
sampled ids out, every step; each step's inputs go up from pinned memory and each step's tokens come
back, the latter while the next step already runs). Inputs larger than L2: every step
reads all weights (~1 GB) and the live requests' cache, several times the 126 MB L2.
"""
from __future__ import annotations

import argparse
import json
import os
import shutil
import statistics
import subprocess
import sys
import tempfile
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

# Layer sizes of the benchmark model: the Qwen2.5-0.5B shape, the reference's headline configuration.
MODEL = {
    "architectures": ["Qwen2ForCausalLM"], "model_type": "qwen2", "num_hidden_layers": 24, "hidden_size": 896,
    "num_attention_heads": 14, "num_key_value_heads": 2, "head_dim": 64, "intermediate_size": 4864,
    "vocab_size": 151936, "rope_theta": 1000000.0, "rms_norm_eps": 1e-6, "tie_word_embeddings": True,
    "max_position_embeddings": 32768, "use_sliding_window": False, "hidden_act": "silu",
    "torch_dtype": "bfloat16",
}
# the other sizes of the family that the baseline names; --shape selects one (the default run is the 0.5B shape)
SHAPES = {
    "0.5b": {},
    "1.5b": {"num_hidden_layers": 28, "hidden_size": 1536, "num_attention_heads": 12, "num_key_value_heads": 2,
             "head_dim": 128, "intermediate_size": 8960},
    "7b": {"num_hidden_layers": 28, "hidden_size": 3584, "num_attention_heads": 28, "num_key_value_heads": 4,
           "head_dim": 128, "intermediate_size": 18944, "vocab_size": 152064, "tie_word_embeddings": False},
}
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0, "source": "fallback"}


def peaks() -> dict:
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.isfile(path):
        try:
            with open(path) as f:
                d = json.load(f)
            out = dict(FALLBACK_PEAKS)
            found = 0
            for k in ("hbm_gbs", "bf16_tflops", "bf16_tflops_sustained"):
                v = d.get(k)
                if isinstance(v, dict):             # {"value": ...} is read as well as a bare number
                    v = v.get("value")
                if isinstance(v, str):
                    v = float(v)
                if isinstance(v, (int, float)) and not isinstance(v, bool) and v > 0:
                    out[k] = float(v)
                    found += 1
            if found:
                out["source"] = "measured" if found == 3 else "measured (partly fallback)"
                return out
        except (OSError, ValueError, AttributeError):
            pass
    return dict(FALLBACK_PEAKS)


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while the timed region runs."""
    FIELDS = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
              "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, index: int = 0):
        self.index, self.proc, self.lines = index, None, []

    def __enter__(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", f"--id={self.index}", f"--query-gpu={self.FIELDS}", "--format=csv,noheader,nounits",
                 "-lms", "20"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            self.thread = threading.Thread(target=self._read, daemon=True)
            self.thread.start()
        except OSError:
            self.proc = None
        return self

    def _read(self):
        for line in self.proc.stdout:
            self.lines.append(line.strip())

    def __exit__(self, *exc):
        if self.proc is not None:
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()

    def summary(self) -> dict:
        sm, mx, reasons = [], [], set()
        names = ("hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap")
        for line in self.lines:
            parts = [p.strip() for p in line.split(",")]
            if len(parts) < 6:
                continue
            try:
                sm.append(float(parts[0]))
                mx.append(float(parts[1]))
            except ValueError:
                continue
            for name, val in zip(names, parts[2:6]):
                if val.lower().startswith("active"):
                    reasons.add(name)
        return {"sm_mhz": statistics.median(sm) if sm else None, "sm_max_mhz": max(mx) if mx else None,
                "reasons": sorted(reasons), "samples": len(sm)}


def model_numbers(layers: int) -> dict:
    """Matrix parameters, bytes a decode step has to read, FLOPs of a prefill, from the sizes."""
    m = MODEL
    h, inter, v = m["hidden_size"], m["intermediate_size"], m["vocab_size"]
    nq, nkv, hd = m["num_attention_heads"], m["num_key_value_heads"], m["head_dim"]
    per_layer = (nq + 2 * nkv) * hd * h + h * nq * hd + 3 * h * inter
    return {
        "kinds": {"qkv": (nq + 2 * nkv) * hd * h, "o_proj": h * nq * hd, "gate_up": 2 * h * inter, "down": h * inter,
                  "lm_head": v * h},
        "attention_flops": lambda t: 4.0 * nq * hd * t * (t + 1) / 2.0,           # one layer, a prompt of t tokens
        "kv_bytes_per_token_layer": 2 * nkv * hd * 2,
        "per_layer_params": per_layer,
        "weight_bytes": 2 * (layers * per_layer + v * h),           # every matrix once, head included
        "kv_bytes_per_token": 2 * layers * nkv * hd * 2,
        "prefill_flops": lambda t: 2.0 * t * layers * per_layer + 2.0 * v * h
        + layers * 4.0 * nq * hd * t * (t + 1) / 2.0,
    }


def _kind_of(kernel: str, what: str, state: dict) -> str:
    """Which part of a layer a launch is, from its kernel and its place in the layer's order: norm, q/k/v,
    (rotation), attention, output projection, norm, gate/up, down."""
    w = what.lower()
    if "attention" in kernel or "attention" in w:
        state["after_attention"] = True
        return "attention"
    if "rmsnorm" in kernel or "rmsnorm" in w:
        return "rmsnorm"
    if "rope" in kernel or "rope" in w:
        return "rope_store"
    if "embed" in kernel or "embed" in w:
        return "embed"
    if "argmax" in kernel or "argmax" in w:
        return "argmax"
    if "gemm" in kernel or "linear" in w or "q/k/v" in w:
        tag = state.get("tag")
        if tag == "swiglu":
            state["after_gate_up"] = True
            return "gate_up"
        if tag == "f32":
            return "lm_head"
        if tag in ("qkv", "store"):
            return "qkv"
        if state.pop("after_attention", False):
            return "o_proj"
        state.pop("after_gate_up", None)
        return "down"
    return kernel or what


def _rows_from_notes(notes):
    """{kind: [microseconds]} and the step's length from the kernels' timer notes: a kernel's share runs from the
    moment its wait for the earlier kernels ended to the moment the next kernel's did."""
    epi = {0: "store", 1: "add", 2: "f32", 3: "swiglu", 4: "qkv"}
    starts = [(t, k, tag) for t, k, tag, phase in notes if phase == 1]
    ends = [t for t, _, _, phase in notes if phase == 2]
    if len(starts) < 2 or not ends:
        return {}, 0.0
    state, rows = {}, {}
    for i, (t, kernel, tag) in enumerate(starts):
        state["tag"] = epi.get(tag) if kernel.startswith("gemm") else None
        kind = _kind_of(kernel, "", state)
        t_next = starts[i + 1][0] if i + 1 < len(starts) else max(ends)
        rows.setdefault(kind, []).append((t_next - t) / 1e3)
    return rows, (max(ends) - starts[0][0]) / 1e3


def decode_breakdown(engine, ops, reqs, rng, vocab, batch, mean_ctx, nums, pk) -> dict:
    """Where the time of ONE decode step goes, from the kernels' own notes of the GPU timer (they keep the overlap
    of dependent launches inside the captured graph): a kernel's share is the time from the moment its wait for the
    earlier kernels ended to the moment the next kernel's did. Bytes: the weights of its product once, or the
    cached keys and values of the live requests; the fraction is of the measured copy bandwidth."""
    import torch
    from nanoinfer_b200.engine import StepEntry
    base = [rc.length for rc in reqs]
    ops.timeline_start()
    engine.reset_graphs()

    def one():
        engine.step([StepEntry(rc, [int(rng.integers(0, vocab))], [0]) for rc in reqs], borrow_logits=True)
    for _ in range(4):
        one()
    ops.timeline_clear()
    one()
    notes = ops.timeline()
    ops.timeline_stop()
    engine.reset_graphs()
    for rc, n in zip(reqs, base):
        engine.truncate(rc, n)
    rows, step_us = _rows_from_notes(notes)
    if not rows:
        return {}
    bytes_of = {k: 2.0 * v for k, v in nums["kinds"].items()}
    bytes_of["attention"] = batch * mean_ctx * nums["kv_bytes_per_token_layer"]
    out = {"step_us": round(step_us, 1)}
    for kind, us in rows.items():
        mean = sum(us) / len(us)
        row = {"n": len(us), "us": round(mean, 2), "share": round(sum(us) / step_us, 3)}
        if kind in bytes_of:
            gbs = bytes_of[kind] / (mean * 1e-6) / 1e9
            row.update({"mb": round(bytes_of[kind] / 1e6, 2), "gbs": round(gbs, 0), "frac": round(gbs / pk["hbm_gbs"], 3)})
        out[kind] = row
    return out


def prefill_breakdown(engine, ops, rng, vocab, t_pre, nums, pk) -> dict:
    """Where the time of one prompt portion goes, from the kernels' own notes of the GPU timer as in
    ``decode_breakdown`` (the third step of the shape: a replay of its captured graph, so the kernels overlap as
    they do in production and the host is not in the way). FLOPs of a product: 2 x tokens x weights; of the
    attention: 4 x heads x head size x t(t+1)/2; the fraction is of the measured cuBLAS burst throughput."""
    import numpy as np
    import torch
    from nanoinfer_b200.engine import StepEntry
    ops.timeline_start()
    engine.reset_graphs()
    rc = engine.open("breakdown")
    ids = rng.integers(0, vocab, t_pre).astype(np.int32)
    for i in range(3):
        if i == 2:
            ops.timeline_clear()
        engine.step([StepEntry(rc, ids, [t_pre - 1])])
        torch.cuda.synchronize()
        engine.truncate(rc, 0)
    notes = ops.timeline()
    ops.timeline_stop()
    engine.reset_graphs()
    engine.close(rc)
    rows, total = _rows_from_notes(notes)
    if not rows:
        return {}
    flops_of = {k: 2.0 * t_pre * v for k, v in nums["kinds"].items()}
    flops_of["lm_head"] = 2.0 * nums["kinds"]["lm_head"]          # one wanted row
    flops_of["attention"] = nums["attention_flops"](t_pre)
    out = {"step_us": round(total, 1)}
    for kind, us in rows.items():
        mean = sum(us) / len(us)
        row = {"n": len(us), "us": round(mean, 2), "share": round(sum(us) / total, 3)}
        if kind in flops_of and kind != "lm_head":
            tf = flops_of[kind] / (mean * 1e-6) / 1e12
            row.update({"gflop": round(flops_of[kind] / 1e9, 2), "tflops": round(tf, 0), "frac": round(tf / pk["bf16_tflops"], 3)})
        out[kind] = row
    return out


def run_ours(args) -> dict:
    import numpy as np
    import torch
    from nanoinfer_b200 import Request, Scheduler, load_model
    from nanoinfer_b200.engine import StepEntry
    from nanoinfer_b200.registry import config_from_json_dict
    from nanoinfer_b200.weights import write_random_model

    pk = peaks()
    layers = args.layers or MODEL["num_hidden_layers"]
    cfg_json = dict(MODEL, num_hidden_layers=layers)
    nums = model_numbers(layers)
    ctx, batch, steps, warmup = args.context, args.batch, args.steps, max(3, args.warmup)
    rng = np.random.default_rng(0)
    vocab = MODEL["vocab_size"]

    tmp = tempfile.mkdtemp(prefix="nanoinfer_b200_bench_")
    t0 = time.time()
    write_random_model(config_from_json_dict(cfg_json), tmp, seed=0)
    max_batch = max(batch, 64)
    page = 16
    num_pages = max_batch * (-(-ctx // page) + 1) + 8
    try:
        model = load_model(tmp, dtype="bfloat16", page_size=page, num_pages=num_pages, max_batch=max_batch,
                           max_tokens_per_step=4096, cuda_graphs=not args.no_graphs)
    finally:
        shutil.rmtree(tmp, ignore_errors=True)      # the weights are on the device now; the folder can be gigabytes
    engine, ops = model.engine, model.engine.rt.ops
    print(f"[bench] model ready in {time.time() - t0:.0f} s", file=sys.stderr, flush=True)
    if args.only == "serve":
        return serve_workload(model, args, rng, vocab, layers)

    def fill(n_req: int, length: int):
        """n_req live requests holding ``length`` random tokens each."""
        reqs = [engine.open(f"b{n_req}_{i}") for i in range(n_req)]
        for rc in reqs:
            done = 0
            while done < length:
                n = min(2048, length - done)
                engine.step([StepEntry(rc, rng.integers(0, vocab, n).tolist(), [])])
                done += n
        return reqs

    def decode_timed(reqs, n_warm: int, n_steps: int, min_seconds: float = 0.5, max_repeats: int = 40):
        """Device time of n_steps decode steps (one token for every request, greedy pick on the device), measured
        again and again FROM THE SAME CONTEXT (the requests forget the n_steps positions in between) until
        min_seconds have been timed. Returns (median ms per step, launches of one region, ms per step of every
        repeat)."""
        out = torch.empty(len(reqs), dtype=torch.int32, device=engine.device)
        toks = [rng.integers(0, vocab, len(reqs)).tolist() for _ in range(n_warm + n_steps)]

        def one(i):
            logits = engine.step([StepEntry(rc, [toks[i][j]], [0]) for j, rc in enumerate(reqs)], borrow_logits=True)
            ops.argmax(logits, out)
        for i in range(n_warm):
            one(i)
        torch.cuda.synchronize()
        base = [rc.length for rc in reqs]
        per_step, launches, total = [], 0, 0.0
        while total < min_seconds * 1e3 and len(per_step) < max_repeats:
            l0 = ops.launches + engine.graph_launches
            start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            start.record()
            for i in range(n_warm, n_warm + n_steps):
                one(i)
            end.record()
            torch.cuda.synchronize()
            ms = start.elapsed_time(end)
            launches = ops.launches + engine.graph_launches - l0
            per_step.append(ms / n_steps)
            total += ms
            for rc, n in zip(reqs, base):
                engine.truncate(rc, n)
        return statistics.median(per_step), launches, per_step

    def close_all(reqs):
        for rc in reqs:
            engine.close(rc)

    # ---- prefill of 2,048 tokens ----------------------------------------------------------
    t_pre = args.prefill_tokens
    pre_ms = []
    for i in range((3 + 7) if args.only != "decode" else 0):
        rc = engine.open(f"p{i}")
        ids = rng.integers(0, vocab, t_pre).astype(np.int32)        # host memory, as a tokenizer's array would be
        torch.cuda.synchronize()
        s, e = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        s.record()
        engine.step([StepEntry(rc, ids, [t_pre - 1])])
        e.record()
        torch.cuda.synchronize()
        if i >= 3:
            pre_ms.append(s.elapsed_time(e))
        engine.close(rc)
    prefill = None
    if pre_ms:
        pre = statistics.median(pre_ms)
        prefill = {"value": round(t_pre / (pre / 1e3), 1), "tokens": t_pre, "ms": round(pre, 3),
                   "frac": round(nums["prefill_flops"](t_pre) / (pre / 1e3) / (pk["bf16_tflops"] * 1e12), 4),
                   "peak": f"{pk['bf16_tflops']:.0f} TFLOP/s, cuBLAS bf16 burst, {pk['source']}"}
    prefill_kernels = None
    if pre_ms and args.breakdown:
        prefill_kernels = prefill_breakdown(engine, ops, rng, vocab, t_pre, nums, pk)

    if args.only == "prefill":
        out = {"impl": "ours", "only": "prefill", "prefill": prefill,
               "config": {"model": f"Qwen2.5-{args.shape.upper()} shape", "layers": layers}}
        if prefill_kernels:
            out["kernels"] = {"prefill": prefill_kernels}
        return out

    # The clocks are sampled from before the warm-up to the end of the timed regions.
    sampler = ClockSampler()
    sampler.__enter__()
    # ---- decode points at batch 1 and 64 --------------------------------------------------
    points = {}
    for b in ((1, 64) if args.only == "all" else ()):
        n_w, n_s = 4, min(steps, 32)
        reqs = fill(b, ctx - n_w - n_s - 1)
        ms, _, _ = decode_timed(reqs, n_w, n_s, min_seconds=0.15)
        points[f"decode_b{b}"] = round(b / (ms / 1e3), 1)
        close_all(reqs)

    # ---- the headline: batch 8 (default), device-timed -------------------------------------
    reqs = fill(batch, ctx - warmup - steps - 1)
    ms_step, launches, repeats = decode_timed(reqs, warmup, steps)
    sampler.__exit__()
    clocks = sampler.summary()
    mean_ctx = ctx - steps / 2.0
    step_bytes = nums["weight_bytes"] + batch * mean_ctx * nums["kv_bytes_per_token"]
    achieved = step_bytes / (ms_step / 1e3) / 1e9
    kernels = None
    if args.breakdown:
        kernels = {"decode": decode_breakdown(engine, ops, reqs, rng, vocab, batch, mean_ctx, nums, pk)}
        if prefill_kernels is not None:
            kernels["prefill"] = prefill_kernels
    close_all(reqs)
    if args.only == "decode":
        out = {"impl": "ours", "only": "decode", "value": round(batch / (ms_step / 1e3), 1), "ms_per_step": round(ms_step, 4),
               "gpu_launches": launches, "repeats": len(repeats), "clocks": clocks,
               "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                            "frac": round(achieved / pk["hbm_gbs"], 4)},
               "config": {"model": f"Qwen2.5-{args.shape.upper()} shape", "layers": layers, "global_batch": batch, "seq_len": ctx}}
        if kernels:
            out["kernels"] = kernels
        return out

    # ---- end to end through the Python entry point (scheduler) -----------------------------
    sched = Scheduler(model, max_batch=batch, max_tokens_per_step=4096, lookahead=True)
    # Requests admitted first decode while the later prompts are still being prefilled (about one step per
    # prompt), so they are ahead by up to `batch` tokens when timing starts; nobody may finish, and nobody may
    # leave the context (and with it the captured graph's bucket), before the timed steps end.
    prompt_len = ctx - warmup - steps - 2 * batch - 8
    for i in range(batch):
        sched.add(Request(f"e{i}", rng.integers(0, vocab, prompt_len).tolist(), max_tokens=ctx))
    while any(s.pending > 1 for s in sched.running) or sched.waiting:
        sched.step()
    for _ in range(warmup):
        sched.step()
    torch.cuda.synchronize()
    t0 = time.perf_counter()
    n_tok = 0
    for _ in range(steps):
        n_tok += len(sched.step().entries)
    torch.cuda.synchronize()
    dt = time.perf_counter() - t0
    h2d = engine.last_h2d_bytes
    for rid in [s.req.request_id for s in sched.running]:
        sched.cancel(rid)
    e2e = {"value": round(n_tok / dt, 1), "unit": "tokens/s", "h2d_bytes_per_step": h2d,
           "d2h_bytes_per_step": 4 * batch, "ms_per_step": round(dt / steps * 1e3, 4)}

    value = batch / (ms_step / 1e3)
    extra = {"kernels": kernels} if kernels else {}
    return {
        **extra,
        "metric": f"decode tok/s at batch {batch} (Qwen2.5-{args.shape.upper()} shape, context {ctx})", "value": round(value, 1),
        "unit": "tokens/s", "n_gpus": 1, "steps": steps, "warmup": warmup, "ms_per_step": round(ms_step, 4),
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16",
        "data": "synthetic: seeded random weights and random token ids", "impl": "ours",
        "config": {"model": f"Qwen2.5-{args.shape.upper()} shape", "layers": layers, "layers_full": MODEL["num_hidden_layers"],
                   "hidden": MODEL["hidden_size"], "heads": MODEL["num_attention_heads"],
                   "kv_heads": MODEL["num_key_value_heads"], "head_dim": MODEL["head_dim"],
                   "intermediate": MODEL["intermediate_size"], "vocab": MODEL["vocab_size"], "tied_head": MODEL["tie_word_embeddings"],
                   "global_batch": batch, "seq_len": ctx, "page_size": page, "prefill_tokens": t_pre,
                   "parallelism": "single-gpu", "l2": f"inputs larger than L2 (weights {nums['weight_bytes'] / 1e9:.1f} GB per step)",
                   "peaks": pk["source"], "timed_regions": len(repeats)},
        "clocks": clocks, "e2e": e2e, "gpu_launches": launches,
        "prefill": prefill,
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4)},
        "points": points,
    }


# ---- another design beside the closest existing one (--design) ------------------------------------------
# Layer sizes that resemble a real model's, small enough for minutes: a Nezalorn stack (delta rule, two gated
# recurrences, latent attention; the last attention layer reads the first one's cached latents) and the Qwen2
# decoder of the same width, depth and vocabulary, with about the same matrix parameters per layer (PolyNorm has
# two feed-forward matrices where SwiGLU has three).
DESIGN_SIZES = {
    "1k": {"width": 1024, "heads": 16, "head_dim": 64, "ff_swiglu": 2816, "rot": 32, "kv_rank": 128, "q_rank": 384,
           "blocks": 8, "window": 1024, "vocab": 32000, "layers": 8},
    "2k": {"width": 2048, "heads": 16, "head_dim": 128, "ff_swiglu": 5632, "rot": 64, "kv_rank": 128, "q_rank": 768,
           "blocks": 16, "window": 1024, "vocab": 32000, "layers": 8},
}


def design_configs(size: dict):
    w, h, d = size["width"], size["heads"], size["head_dim"]
    ff = {"kind": "dense", "ff": size["ff_swiglu"] * 3 // 2}
    lat = {"heads": h, "dim": d, "rot_dim": size["rot"], "vdim": d, "q_rank": size["q_rank"], "kv_rank": size["kv_rank"],
           "mask": {"size": size["window"]}, "scale": (d + size["rot"]) ** -0.5,
           "rot": {"dims": size["rot"], "base": 10000.0, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    delta = {"type": "general_delta", "mixer": {"heads": h, "dim": d, "decay_rank": 64}, "mlp": ff}
    lru = {"type": "rglru", "mixer": {"width": w, "conv": 4, "blocks": size["blocks"]}, "mlp": ff}
    layers = []
    for i in range(size["layers"]):
        kind = i % 4
        if kind == 0:
            layers.append(delta)
        elif kind in (1, 2):
            layers.append(lru)
        else:
            m = dict(lat) if i == 3 else dict(lat, kv_from=3)
            layers.append({"type": "latent_attention", "mixer": m, "mlp": ff})
    nez = {"architecture": "Nezalorn", "vocab": size["vocab"], "width": w, "norm": {"eps": 1e-5}, "layers": layers}
    qwen = {"architectures": ["Qwen2ForCausalLM"], "model_type": "qwen2", "num_hidden_layers": size["layers"], "hidden_size": w,
            "num_attention_heads": h, "num_key_value_heads": 2, "head_dim": d, "intermediate_size": size["ff_swiglu"],
            "vocab_size": size["vocab"], "rope_theta": 1000000.0, "rms_norm_eps": 1e-6, "tie_word_embeddings": True,
            "max_position_embeddings": 32768, "use_sliding_window": False, "hidden_act": "silu", "torch_dtype": "bfloat16"}
    return nez, qwen


# A Vafozen stack at the same widths: chunked softmax attention beside gated linear attention, a state-space mixer,
# rotated and capped softmax attention beside a time mix, a state-space mixer, twice; SwiGLU feed-forwards of the Qwen2
# decoder's size; the softmax halves have the Qwen2 decoder's head counts and head size.
VAFOZEN_SIZES = {
    "1k": {"width": 1024, "heads": 16, "head_dim": 64, "ff_swiglu": 2816, "rot": 32, "side_heads": 4, "decay_rank": 64,
           "ssm_heads": 32, "ssm_state": 128, "chunk": 1024, "vocab": 32000, "layers": 8},
    "2k": {"width": 2048, "heads": 16, "head_dim": 128, "ff_swiglu": 5632, "rot": 64, "side_heads": 4, "decay_rank": 64,
           "ssm_heads": 32, "ssm_state": 128, "chunk": 1024, "vocab": 32000, "layers": 8},
}


def vafozen_configs(size: dict):
    w, h, d = size["width"], size["heads"], size["head_dim"]
    ff = {"kind": "dense", "ff": size["ff_swiglu"]}
    side = {"heads": size["side_heads"], "dim": d, "decay_rank": size["decay_rank"]}
    chunked = {"heads": h, "kv_heads": 2, "dim": d, "vdim": d, "scale": d ** -0.5, "mask": {"size": size["chunk"]}}
    rotated = {"heads": h, "kv_heads": 2, "dim": d, "vdim": d, "scale": d ** -0.5, "conv": 4, "softcap": 30.0,
               "rot": {"dims": size["rot"], "base": 10000.0}}
    kinds = [
        {"type": "parallel", "mixer": {"left": chunked, "right": dict(side, tau=16.0), "left_scale": 1.0, "right_scale": 1.0}, "mlp": ff},
        {"type": "mamba2", "mixer": {"heads": size["ssm_heads"], "vdim": 2 * w // size["ssm_heads"], "state": size["ssm_state"], "groups": 2,
                                     "norm_groups": 2, "conv": 4}, "mlp": ff},
        {"type": "parallel_2", "mixer": {"left": rotated, "right": dict(side), "left_scale": 1.0, "right_scale": 1.0}, "mlp": ff},
    ]
    layers = [kinds[(0, 1, 2, 1)[i % 4]] for i in range(size["layers"])]
    vaf = {"architecture": "Vafozen", "vocab": size["vocab"], "width": w, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0}, "layers": layers}
    return vaf, design_configs(dict(DESIGN_SIZES["1k"], **{k: size[k] for k in ("width", "heads", "head_dim", "ff_swiglu", "vocab", "layers")}))[1]


# A Darotar stack at the same widths: attention through a latent (sink, output gate; every second such layer reads the
# rows of the one before) and windowed attention whose values are the keys, by turns; every feed-forward is a mixture of
# 8 experts of which a token uses 2, each half as wide as the Qwen2 decoder's feed-forward, so that a token passes through
# as many feed-forward parameters in both models. The attention layers have the Qwen2 decoder's head counts and head size.
DAROTAR_SIZES = {
    "1k": {"width": 1024, "heads": 16, "head_dim": 64, "ff_swiglu": 2816, "rot": 32, "kv_rank": 128, "q_rank": 384,
           "experts": 8, "top": 2, "window": 1024, "vocab": 32000, "layers": 8},
    "2k": {"width": 2048, "heads": 16, "head_dim": 128, "ff_swiglu": 5632, "rot": 64, "kv_rank": 128, "q_rank": 768,
           "experts": 8, "top": 2, "window": 1024, "vocab": 32000, "layers": 8},
}


def darotar_configs(size: dict):
    w, h, d = size["width"], size["heads"], size["head_dim"]
    ff = {"kind": "moe", "expert": {"ff": size["ff_swiglu"] // size["top"]}, "router": {"experts": size["experts"], "top": size["top"]}}
    lat = {"heads": h, "dim": d, "rot_dim": size["rot"], "vdim": d, "q_rank": size["q_rank"], "kv_rank": size["kv_rank"],
           "scale": (d + size["rot"]) ** -0.5, "rot": {"dims": size["rot"], "base": 10000.0}}
    att = {"heads": h, "kv_heads": 2, "dim": d, "vdim": d, "scale": 8.0 / d, "mask": {"size": size["window"]},
           "rot": {"dims": d, "base": 10000.0, "scaling": {"factor": 2.0}}}
    layers = []
    for i in range(size["layers"]):
        if i % 2:
            layers.append({"type": "attention", "mixer": att, "mlp": ff})
        else:
            layers.append({"type": "latent_attention", "mixer": dict(lat, kv_from=i - 2) if i % 4 == 2 else dict(lat), "mlp": ff})
    dar = {"architecture": "Darotar", "vocab": size["vocab"], "width": w, "norm": {"eps": 1e-5}, "residual_mult": 0.5, "layers": layers}
    return dar, design_configs(dict(DESIGN_SIZES["1k"], **{k: size[k] for k in ("width", "heads", "head_dim", "ff_swiglu", "vocab", "layers")}))[1]


# A Dusilorn stack at the same widths: rotated attention behind a sliding window and chunked attention with a sink and a
# norm of q and k over the whole projection, by turns, all with the Qwen2 decoder's head counts and head size and with
# blended values; the first feed-forward dense, the others mixtures of 8 experts without a gate (relu squared, two
# matrices each) and one identity output, of which a token uses 2, beside a shared expert: the chosen experts and the
# shared one are half as wide as the Qwen2 decoder's feed-forward each, so a token passes through as many feed-forward
# parameters in both models (2 x 2 + 2 halves against 3 matrices).
DUSILORN_SIZES = {
    "1k": {"width": 1024, "heads": 16, "head_dim": 64, "ff_swiglu": 2816, "rot": 32, "experts": 8, "identity": 1, "top": 2,
           "window": 1024, "vocab": 32000, "layers": 8},
    "2k": {"width": 2048, "heads": 16, "head_dim": 128, "ff_swiglu": 5632, "rot": 64, "experts": 8, "identity": 1, "top": 2,
           "window": 1024, "vocab": 32000, "layers": 8},
}


def dusilorn_configs(size: dict):
    w, h, d = size["width"], size["heads"], size["head_dim"]
    half = size["ff_swiglu"] // 2
    ff = {"kind": "moe", "expert": {"ff": half}, "router": {"experts": size["experts"], "identity": size["identity"], "top": size["top"]},
          "shared": {"ff": half}}
    common = {"heads": h, "kv_heads": 2, "dim": d, "vdim": d, "scale": d ** -0.5, "softcap": 30.0, "v_mix": True, "mask": {"size": size["window"]}}
    layers = []
    for i in range(size["layers"]):
        mlp = {"kind": "dense", "ff": size["ff_swiglu"]} if i == 0 else ff
        if i % 2:
            layers.append({"type": "attention", "mixer": dict(common), "mlp": mlp})
        else:
            layers.append({"type": "attention_2", "mixer": dict(common, rot={"dims": size["rot"], "base": 1000000.0}), "mlp": mlp})
    dus = {"architecture": "Dusilorn", "vocab": size["vocab"], "width": w, "norm": {"eps": 1e-5}, "embedding": {"scale": 8.0},
           "logit_scale": 0.5, "layers": layers}
    return dus, design_configs(dict(DESIGN_SIZES["1k"], **{k: size[k] for k in ("width", "heads", "head_dim", "ff_swiglu", "vocab", "layers")}))[1]


# A Pilonex stack at the same widths, two residual streams: six layers of which the first two run twice (eight layer runs, as many
# as the Qwen2 decoder has layers): windowed attention with the Qwen2 decoder's head counts and head size beside a gated
# delta rule, and matrix memories. Feed-forwards of the clamped gated form by turns dense, as wide as the Qwen2 decoder's,
# and mixtures of 8 experts of which a token uses 2, each half as wide.
PILONEX_SIZES = {
    "1k": {"width": 1024, "heads": 16, "head_dim": 64, "ff_swiglu": 2816, "delta_heads": 8, "rank": 64, "memory_heads": 8, "experts": 8, "top": 2,
           "window": 1024, "streams": 2, "vocab": 32000, "layers": 8},
    "2k": {"width": 2048, "heads": 16, "head_dim": 128, "ff_swiglu": 5632, "delta_heads": 8, "rank": 64, "memory_heads": 8, "experts": 8, "top": 2,
           "window": 1024, "streams": 2, "vocab": 32000, "layers": 8},
}


def pilonex_configs(size: dict):
    h, d, n = size["heads"], size["head_dim"], size["delta_heads"]
    dense = {"kind": "dense", "ff": size["ff_swiglu"], "limit": 7.0}
    routed = {"kind": "moe", "expert": {"ff": size["ff_swiglu"] // size["top"], "limit": 7.0}, "router": {"experts": size["experts"], "top": size["top"]}}
    pair = {"left": {"heads": h, "kv_heads": 2, "dim": d, "vdim": d, "scale": d ** -0.5, "mask": {"size": size["window"]},
                     "rot": {"dims": d, "base": 500000.0, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 4096}}},
            "right": {"heads": n, "kv_heads": n, "dim": d, "vdim": d, "conv": 4, "decay_rank": size["rank"], "gate_rank": size["rank"]},
            "left_scale": 1.0, "right_scale": 0.75}
    memory = {"heads": size["memory_heads"], "dim": d, "vdim": size["width"] // size["memory_heads"], "gate_cap": 15.0}
    order = [("parallel", dense), ("parallel", routed), ("mlstm", dense), ("parallel", routed), ("mlstm", dense), ("parallel", routed)]
    layers = [{"type": t, "mixer": pair if t == "parallel" else memory, "mlp": mlp} for t, mlp in order]
    pil = {"architecture": "Pilonex", "vocab": size["vocab"], "width": size["width"], "norm": {"eps": 1e-5}, "streams": size["streams"],
           "loop": {"start": 0, "stop": 2, "times": 2}, "layers": layers}
    return pil, design_configs(dict(DESIGN_SIZES["1k"], **{k: size[k] for k in ("width", "heads", "head_dim", "ff_swiglu", "vocab", "layers")}))[1]


# A Vagulorn stack at the same widths, layer for layer like the Vafozen stack: softmax attention whose values are its keys (a sliding
# window beside four kept tokens, a gate per head) beside lightning attention, a state-space mixer, chunked attention, a state-space
# mixer, twice; gelu-gated feed-forwards of the Qwen2 decoder's size; the softmax mixers have the Qwen2 decoder's head counts and head
# size. Its closest existing model is Vafozen (parallel blocks with one norm, a pair of mixers, the same state-space mixer).
VAGULORN_SIZES = {name: dict({k: v for k, v in size.items() if k != "decay_rank"}, window=1024, keep_first=4)
                  for name, size in VAFOZEN_SIZES.items()}


def vagulorn_configs(size: dict):
    w, h, d, n = size["width"], size["heads"], size["head_dim"], size["side_heads"]
    ff = {"kind": "dense", "ff": size["ff_swiglu"]}
    half = {"heads": h, "kv_heads": 2, "dim": d, "vdim": d, "scale": d ** -0.5}
    pair = {"left": dict(half, mask={"size": size["window"], "keep_first": size["keep_first"]}, rot={"dims": size["rot"], "base": 500000.0}),
            "right": {"heads": n, "dim": d, "vdim": d, "decay": [1.0 - 2.0 ** -(3 + 2 * i) for i in range(n)]}, "left_scale": 1.0, "right_scale": 0.75}
    chunked = dict(half, mask={"size": size["chunk"]}, rot={"dims": size["rot"], "base": 50000.0})
    ssm = {"heads": size["ssm_heads"], "vdim": 2 * w // size["ssm_heads"], "state": size["ssm_state"], "groups": 2, "norm_groups": 2, "conv": 4}
    kinds = [{"type": "parallel", "mixer": pair, "mlp": ff}, {"type": "mamba2", "mixer": ssm, "mlp": ff}, {"type": "attention", "mixer": chunked, "mlp": ff}]
    layers = [kinds[(0, 1, 2, 1)[i % 4]] for i in range(size["layers"])]
    vag = {"architecture": "Vagulorn", "vocab": size["vocab"], "width": w, "norm": {"eps": 1e-5}, "embedding": {"scale": 8.0}, "layers": layers}
    return (vag,) + vafozen_configs(dict(size, decay_rank=64))


def run_design(args) -> dict:
    """Prefill and decode throughput of a design (Nezalorn, Vafozen, Darotar, Dusilorn, Pilonex, Vagulorn) beside the Qwen2 decoder at equal
    size (Vagulorn: beside Vafozen as well; random weights, bfloat16, device-timed with CUDA events), and where one eager step's time goes,
    launch kind by launch kind."""
    import numpy as np
    import torch
    from nanoinfer_b200 import load_model
    from nanoinfer_b200.engine import StepEntry
    from nanoinfer_b200.registry import config_from_json_dict
    from nanoinfer_b200.weights import write_random_model
    pk = peaks()
    t_pre, batch, ctx = args.prefill_tokens, args.batch, min(args.context, 2048)
    steps, warmup = min(args.steps, 64), max(3, args.warmup)
    design = args.design
    sizes, configs = {"nezalorn": (DESIGN_SIZES, design_configs), "vafozen": (VAFOZEN_SIZES, vafozen_configs),
                      "darotar": (DAROTAR_SIZES, darotar_configs), "dusilorn": (DUSILORN_SIZES, dusilorn_configs),
                      "pilonex": (PILONEX_SIZES, pilonex_configs), "vagulorn": (VAGULORN_SIZES, vagulorn_configs)}[design]
    beside = ("vafozen", "qwen2") if design == "vagulorn" else ("qwen2",)
    out = {"impl": "ours", "design": design, "dtype": "bf16", "data": "synthetic: seeded random weights and random token ids",
           "peaks": {"hbm_gbs": pk["hbm_gbs"], "bf16_tflops": pk["bf16_tflops"], "source": pk["source"]},
           "config": {"prefill_tokens": t_pre, "decode_batch": batch, "decode_context": ctx, "page_size": 16}, "sizes": {}}
    for name in (args.design_sizes.split(",") if args.design_sizes else sorted(sizes)):
        size = sizes[name]
        row = {}
        for label, cfg_json in zip((design,) + beside, configs(size)):
            rng = np.random.default_rng(0)
            tmp = tempfile.mkdtemp(prefix="nanoinfer_b200_design_")
            try:
                write_random_model(config_from_json_dict(cfg_json), tmp, seed=0)
                model = load_model(tmp, dtype="bfloat16", page_size=16, num_pages=(batch + 1) * (ctx // 16 + 8) + t_pre // 16 + 8,
                                   max_batch=batch + 1, max_tokens_per_step=4096, cuda_graphs=not args.no_graphs)
            finally:
                shutil.rmtree(tmp, ignore_errors=True)
            engine, ops, vocab = model.engine, model.engine.rt.ops, size["vocab"]

            def timed(fn, n):
                torch.cuda.synchronize()
                s, e = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                s.record()
                for _ in range(n):
                    fn()
                e.record()
                torch.cuda.synchronize()
                return s.elapsed_time(e) / n

            # prefill: one prompt of t_pre tokens, logits of the last (3 warm-up prompts, the median of 7)
            pre = []
            for i in range(10):
                rc = engine.open(f"p{i}")
                ids = rng.integers(0, vocab, t_pre).astype(np.int32)
                ms = timed(lambda: engine.step([StepEntry(rc, ids, [t_pre - 1])]), 1)
                engine.close(rc)
                if i >= 3:
                    pre.append(ms)
            # decode: `batch` requests holding ctx tokens each go on token by token (contexts grow by `steps`)
            reqs = [engine.open(f"d{i}") for i in range(batch)]
            for rc in reqs:
                done = 0
                while done < ctx - warmup - steps:
                    n = min(2048, ctx - warmup - steps - done)
                    engine.step([StepEntry(rc, rng.integers(0, vocab, n).astype(np.int32), [])])
                    done += n
            pick = torch.empty(batch, dtype=torch.int32, device=engine.device)

            def one():
                logits = engine.step([StepEntry(rc, [int(rng.integers(0, vocab))], [0]) for rc in reqs], borrow_logits=True)
                ops.argmax(logits, pick)
            for _ in range(warmup):
                one()
            l0 = ops.launches + engine.graph_launches
            with ClockSampler() as cs:
                dec_ms = timed(one, steps)
            launches = ops.launches + engine.graph_launches - l0
            # where the time goes: one eager prompt and one eager decode step with an event behind every launch
            kinds = {}
            if args.breakdown:
                eager = ops
                for phase in ("prefill", "decode"):
                    if phase == "prefill":
                        rc = engine.open("t")
                        ids = rng.integers(0, vocab, t_pre).astype(np.int32)
                        entries = [StepEntry(rc, ids, [t_pre - 1])]
                    else:
                        entries = [StepEntry(rc, [int(rng.integers(0, vocab))], [0]) for rc in reqs]
                    graphs = (engine._graphs, engine._portion_graphs)
                    engine._graphs = engine._portion_graphs = None
                    try:
                        eager.time_ops(True)
                        engine.step(entries)
                        agg = {}
                        for what, us in eager.op_times():
                            n, tot = agg.get(what, (0, 0.0))
                            agg[what] = (n + 1, tot + us)
                        eager.time_ops(False)
                    finally:
                        engine._graphs, engine._portion_graphs = graphs
                    kinds[phase] = {k: {"n": n, "us": round(t, 1)} for k, (n, t) in sorted(agg.items(), key=lambda kv: -kv[1][1])}
                    if phase == "prefill":
                        engine.close(rc)
            for rc in reqs:
                engine.close(rc)
            pre_ms = statistics.median(pre)
            row[label] = {"prefill_ms": round(pre_ms, 3), "prefill_tok_s": round(t_pre / pre_ms * 1e3, 1),
                          "decode_ms_per_step": round(dec_ms, 4), "decode_tok_s": round(batch / dec_ms * 1e3, 1),
                          "weight_bytes": model.weight_bytes()[0], "decode_launches": launches, "clocks": cs.summary()}
            if kinds:
                row[label]["launch_kinds_us"] = kinds
            del model, engine, ops
            torch.cuda.empty_cache()
        for other in beside:        # the keys without a name are the ratios to the dense decoder
            name_of = "" if other == "qwen2" else f"_{other}"
            row["ratio_prefill" + name_of] = round(row[design]["prefill_tok_s"] / row[other]["prefill_tok_s"], 3)
            row["ratio_decode" + name_of] = round(row[design]["decode_tok_s"] / row[other]["decode_tok_s"], 3)
        out["sizes"][name] = dict(row, size=size)
    return out


def serve_workload(model, args, rng, vocab: int, layers: int) -> dict:
    """A mixed continuous batch through the scheduler: 64 requests with prompts of 128 to 2,048 random ids
    and 256 decoded tokens each, all queued at once; prompts are cut under a budget of 2,048 tokens a step
    and run beside the decoding requests. Wall-clock time from the first step to the last token, host ids in
    and sampled ids out; the first run warms up (it captures the decode graphs), the second is timed."""
    import torch
    from nanoinfer_b200 import Request, Scheduler
    n_req, new_tokens, budget = 64, 256, 2048
    lens = rng.integers(128, 2049, n_req)

    def run():
        sched = Scheduler(model, max_batch=n_req, max_tokens_per_step=budget, lookahead=True)
        for i, n in enumerate(lens):
            sched.add(Request(f"r{i}", rng.integers(0, vocab, int(n)).tolist(), max_tokens=new_tokens))
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        t_prompts, steps_prompts = None, 0
        while sched.has_work():
            plan = sched.step()
            if t_prompts is None and not sched.waiting and all(e.count == 1 for e in plan.entries):
                torch.cuda.synchronize()            # every prompt is in the cache: the rest is decoding
                t_prompts, steps_prompts = time.perf_counter() - t0, sched.steps
        torch.cuda.synchronize()
        dt = time.perf_counter() - t0
        generated = sum(len(v) for v in sched.finished.values())
        return dt, generated, sched.steps, t_prompts, steps_prompts, sched.preemptions

    run()
    dt, generated, steps, t_prompts, steps_prompts, preemptions = run()
    return {"impl": "ours", "only": "serve", "metric": "generated tok/s of a continuous batch (64 requests, prompts 128-2048, 256 new tokens each)",
            "value": round(generated / dt, 1), "unit": "tokens/s", "ms_total": round(dt * 1e3, 1), "steps": steps,
            "total_tokens_per_s": round((generated + int(lens.sum())) / dt, 1),
            "prompt_phase_ms": round(t_prompts * 1e3, 1), "prompt_phase_steps": steps_prompts,
            "decode_ms_per_step": round((dt - t_prompts) * 1e3 / max(1, steps - steps_prompts), 4),
            "preemptions": preemptions,
            "config": {"model": f"Qwen2.5-{args.shape.upper()} shape", "layers": layers, "requests": n_req,
                       "prompt_tokens": int(lens.sum()), "new_tokens": new_tokens, "max_tokens_per_step": budget,
                       "page_size": 16}}


def run_reference(args) -> dict:
    """The unmodified reference (its Python model, installed under baseline/_ref) on the same workload:
    random weights of the same shape, batch 8 decode at context 4096 through ``Model.forward`` with its
    ``KVCache`` and ``sample_next_token``, the calls its own generate loop makes (nanoinfer/generate.py:72-83)."""
    ref_dir = os.path.join(ROOT, "baseline", "_ref")
    if not os.path.isdir(os.path.join(ref_dir, "nanoinfer")):
        return {"impl": "reference", "unavailable": "baseline/_ref/nanoinfer is not installed (pip install --no-deps --target baseline/_ref <reference>)"}
    sys.path.insert(0, ref_dir)
    try:
        import torch
        from nanoinfer.config import ModelConfig
        from nanoinfer.model import Model
        from nanoinfer.sampling import SamplingParams, sample_next_token
    except Exception as e:  # noqa: BLE001
        return {"impl": "reference", "unavailable": f"cannot import the reference: {type(e).__name__}: {e}"}
    if not torch.cuda.is_available():
        return {"impl": "reference", "unavailable": "no CUDA device"}
    m = MODEL
    layers = args.layers or m["num_hidden_layers"]
    ctx, batch, steps, warmup = args.context, args.batch, args.steps, max(3, args.warmup)
    cfg = ModelConfig(vocab_size=m["vocab_size"], hidden_size=m["hidden_size"], intermediate_size=m["intermediate_size"],
                      num_layers=layers, num_attention_heads=m["num_attention_heads"],
                      num_kv_heads=m["num_key_value_heads"], head_dim=m["head_dim"], rms_norm_eps=m["rms_norm_eps"],
                      rope_theta=m["rope_theta"], max_position_embeddings=m["max_position_embeddings"],
                      tie_word_embeddings=True)
    torch.manual_seed(0)
    model = Model(cfg).to(device="cuda", dtype=torch.bfloat16).eval()
    model.lm_head.weight = model.embed_tokens.weight
    cache = model.init_cache(batch, ctx)
    g = torch.Generator(device="cpu").manual_seed(0)
    filled, target = 0, ctx - warmup - steps - 1
    with torch.no_grad():
        while filled < target:
            n = min(512, target - filled)
            model(torch.randint(0, m["vocab_size"], (batch, n), generator=g).cuda(), cache=cache)
            filled += n
        params = SamplingParams()
        pinned = torch.empty((batch, 1), dtype=torch.long).pin_memory()

        def one():
            pinned.copy_(torch.randint(0, m["vocab_size"], (batch, 1), generator=g))
            cur = pinned.to("cuda", non_blocking=True)
            logits = model(cur, cache=cache)[:, -1, :]
            return [sample_next_token(logits[b], params) for b in range(batch)]
        for _ in range(warmup):
            one()
        torch.cuda.synchronize()
        s, e = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        with ClockSampler() as cs:
            t0 = time.perf_counter()
            s.record()
            for _ in range(steps):
                one()
            e.record()
            torch.cuda.synchronize()
            dt = time.perf_counter() - t0
        ms = s.elapsed_time(e) / steps
    return {
        "metric": "decode tok/s at batch 8 (Qwen2.5-0.5B shape, context 4096)", "value": round(batch / (ms / 1e3), 1),
        "unit": "tokens/s", "n_gpus": 1, "steps": steps, "warmup": warmup, "ms_per_step": round(ms, 4),
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16",
        "data": "synthetic: random weights and random token ids", "impl": "reference",
        "config": {"model": f"Qwen2.5-{args.shape.upper()} shape", "layers": layers, "layers_full": m["num_hidden_layers"],
                   "hidden": m["hidden_size"], "heads": m["num_attention_heads"], "kv_heads": m["num_key_value_heads"],
                   "head_dim": m["head_dim"], "intermediate": m["intermediate_size"], "vocab": m["vocab_size"],
                   "tied_head": m["tie_word_embeddings"], "global_batch": batch, "seq_len": ctx, "page_size": 16,
                   "prefill_tokens": args.prefill_tokens, "parallelism": "single-gpu",
                   "l2": "inputs larger than L2 (weights 1.0 GB per step)", "peaks": peaks()["source"], "timed_regions": 1},
        "engine": "reference Python model (torch, CUDA)",
        "clocks": cs.summary(),
        "e2e": {"value": round(batch * steps / dt, 1), "unit": "tokens/s", "h2d_bytes_per_step": 8 * batch,
                "d2h_bytes_per_step": 8 * batch},
        "gpu_launches": 0,
    }


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=128)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--context", type=int, default=4096)
    ap.add_argument("--prefill-tokens", type=int, default=2048)
    ap.add_argument("--layers", type=int, default=0, help="fewer layers than the model has (0 = all)")
    ap.add_argument("--no-graphs", action="store_true", help="launch decode steps kernel by kernel (for profilers that filter by kernel name)")
    ap.add_argument("--only", default="all", choices=["all", "prefill", "decode", "serve"],
                    help="measure one part only (for profiling small cases); the JSON line then lacks the rest. "
                         "'serve' runs the continuous-batching workload (64 requests through the scheduler) instead")
    ap.add_argument("--breakdown", action="store_true",
                    help="add a 'kernels' block: where the time of a decode step and of a prompt portion goes, kernel kind by "
                         "kind, with bytes or FLOPs and the fraction of the measured peak")
    ap.add_argument("--shape", default="0.5b", choices=sorted(SHAPES), help="layer sizes: the family's 0.5B (default), 1.5B or 7B")
    ap.add_argument("--design", default=None, choices=["nezalorn", "vafozen", "darotar", "dusilorn", "pilonex", "vagulorn"],
                    help="instead of the headline workload: prefill and decode throughput of this design beside the Qwen2 "
                         "decoder at equal size (--design-sizes, --prefill-tokens, --batch, --context up to 2048, --breakdown)")
    ap.add_argument("--design-sizes", default="", help="comma-separated names of DESIGN_SIZES (default: all)")
    args = ap.parse_args()
    MODEL.update(SHAPES[args.shape])
    if args.gpus != 1 or int(os.environ.get("WORLD_SIZE", "1")) > 1:
        if int(os.environ.get("RANK", "0")) == 0:
            print(json.dumps({"unavailable": f"this engine runs on one GPU; --gpus {args.gpus} is not supported",
                              "n_gpus": args.gpus}))
        return 2
    if args.steps + args.warmup + 2 >= args.context:
        print(json.dumps({"unavailable": "steps + warmup must be smaller than the context"}))
        return 2
    if args.design and args.impl == "ours":
        print(json.dumps(run_design(args)), flush=True)
        return 0
    result = run_reference(args) if args.impl == "reference" else run_ours(args)
    print(json.dumps(result), flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
