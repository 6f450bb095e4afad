"""Benchmark of the serving step: decode tokens/s and prefill tokens/s of a
Qwen2.5-7B-shaped model with random weights on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference]

A "step" is one decode step of a batch of 8 requests whose prompts of 2,048 tokens are
already cached (context 2,048 + tokens decoded so far, inside the benchmark context of
4,096).  It prints ONE JSON line:

  value            decoded tokens/s of the timed K steps, timed on the device with CUDA
                   events (host tokens chosen beforehand, sampling kernel included)
  e2e              the same through the Python entry point (Engine.step): every step
                   uploads its integer arrays from pinned host memory and reads the sampled
                   ids back to the host
  prefill          one prompt of 2,048 tokens in one step: tokens/s, ms, fraction of the
                   bf16 peak that its flops reach
  roofline         bytes the decode step must read (every weight once + the cache of the
                   live requests) / its time, against the HBM peak
  points           decode tokens/s at batch 1 and 64; at contexts of 8,192 and 32,768 tokens (batch 1 and 8); and at
                   the 14B and 32B shapes of the same architecture (batch 8, 2,048-token prompts), each with its
                   fraction of the copy roofline (`hbm_frac_*`)
  kernels          per workload (decode at batch 1, 8 and 64, the 2,048-token prefill) and kernel class
                   (norm, qkv, rotary+write, attention, o, gate_up, down, head, sampler): device
                   microseconds with every kernel alone (CUDA events between the launches of an
                   eager step), the bytes or flops the class has to do, and the fraction of the
                   measured peak; ``sum_over_step`` compares the classes' sum with that step's time
  env              GPU, compute capability, torch and CUDA versions, commit, time

Peaks come from MEASURED_PEAKS.json beside this file if it is there, else from the
fallback figures (6.65 TB/s copy bandwidth, 1.59 PFLOP/s bf16).  Every step streams
15 GB of weights, far more than the 126 MB of L2, so no separate L2 flush is needed.
"""

from __future__ import annotations

import argparse
import json
import subprocess
import sys
import threading
import time
from pathlib import Path

ROOT = Path(__file__).resolve().parent
sys.path.insert(0, str(ROOT))

# the headline configuration: the Qwen2.5-7B shape
CONFIG_7B = dict(architectures=["Qwen2ForCausalLM"], hidden_size=3584, intermediate_size=18944,
                 num_hidden_layers=28, num_attention_heads=28, num_key_value_heads=4, head_dim=128,
                 vocab_size=152064, rope_theta=1e6, rms_norm_eps=1e-6, tie_word_embeddings=False,
                 max_position_embeddings=32768)
PROMPT_LEN = 2048
CONTEXT = 4096
PAGE_SIZE = 16
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0}


# Decode steps run untimed before the W warm-up steps of a decode measurement: the prompts before them are a burst of
# dense products that leaves the SM clock low under the power cap for a while, and a decode step measured right after
# it reads 2-3 % slower than the same step a tenth of a second later.
SETTLE_STEPS = 32


def load_peaks():
    p = ROOT / "MEASURED_PEAKS.json"
    if p.is_file():
        try:
            raw = json.loads(p.read_text())
            return {"hbm_gbs": float(raw["hbm_gbs"]), "bf16_tflops": float(raw["bf16_tflops"]),
                    "bf16_tflops_sustained": float(raw.get("bf16_tflops_sustained", raw["bf16_tflops"])),
                    "source": "measured"}
        except (KeyError, ValueError, TypeError):
            pass
    return dict(FALLBACK_PEAKS, source="fallback")


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while the timed region runs."""

    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, index: int = 0):
        self.index, self.rows, self.proc, self.thread = index, [], None, None

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", f"--id={self.index}", f"--query-gpu={self.QUERY}",
                                          "--format=csv,noheader,nounits", "-lms", "50"],
                                         stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
        except OSError:
            return
        self.thread = threading.Thread(target=self._read, daemon=True)
        self.thread.start()

    def _read(self):
        for line in self.proc.stdout:
            self.rows.append([c.strip() for c in line.split(",")])

    def mark(self) -> int:
        return len(self.rows)

    def stop(self):
        if self.proc is not None:
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()

    def summary(self, lo: int = 0, hi: "int | None" = None) -> dict:
        rows = [r for r in self.rows[lo:hi] if len(r) == 6] or [r for r in self.rows if len(r) == 6]
        if not rows:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["unavailable"]}
        mhz = sorted(int(r[0]) for r in rows if r[0].isdigit())
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = [n for i, n in enumerate(names) if any(r[2 + i].lower().startswith("active") for r in rows)]
        return {"sm_mhz": mhz[len(mhz) // 2] if mhz else None,
                "sm_max_mhz": int(rows[0][1]) if rows[0][1].isdigit() else None, "reasons": reasons,
                "samples": len(rows)}


def bench_config(cfg_raw: dict, layers: int, layers_full: int, batch: int) -> dict:
    """The ``config`` block of the bench line: every size of the measured model and workload, flat.
    Both arms (this engine and the reference) print the same keys with the same values."""
    return {"model": "Qwen2.5-7B-shaped, random weights", "layers": layers, "layers_full": layers_full,
            "hidden": cfg_raw["hidden_size"], "heads": cfg_raw["num_attention_heads"],
            "kv_heads": cfg_raw["num_key_value_heads"], "head_dim": cfg_raw["head_dim"],
            "intermediate": cfg_raw["intermediate_size"], "vocab": cfg_raw["vocab_size"],
            "global_batch": batch, "seq_len": CONTEXT, "prompt_len": PROMPT_LEN, "page_size": PAGE_SIZE,
            "parallelism": "single GPU", "l2": "inputs larger than L2 (15 GB of weights per step)"}


def model_numbers(cfg: dict, layers: int):
    """Weight bytes a decode step reads, cache bytes per token, and flops of a step of T tokens."""
    H, I, V = cfg["hidden_size"], cfg["intermediate_size"], cfg["vocab_size"]
    nh, nkv, hd = cfg["num_attention_heads"], cfg["num_key_value_heads"], cfg["head_dim"]
    per_layer = H * (nh + 2 * nkv) * hd + nh * hd * H + 3 * H * I
    small = layers * (2 * H + (nh + 2 * nkv) * hd) * 4 + H * 4
    weight_bytes = (layers * per_layer + V * H) * 2 + small
    kv_bytes_per_token = layers * 2 * nkv * hd * 2

    def flops(T: int, context_start: int, logit_rows: int) -> float:
        linear = 2.0 * T * layers * per_layer
        # causal attention of T new tokens over context_start cached ones: QK^T and PV
        keys = T * context_start + T * (T + 1) / 2
        attn = 4.0 * layers * nh * hd * keys
        return linear + attn + 2.0 * logit_rows * H * V
    return weight_bytes, kv_bytes_per_token, flops


def class_work(cfg: dict, layers: int, T: int, B: int, context_before: int, logit_rows: int) -> dict:
    """Per kernel class of one step (T tokens in B entries, each with ``context_before`` tokens cached): the
    bytes it has to move and the flops it has to do, summed over the layers.  Bytes: every weight once, the
    cache of the live requests once, activations in and out once (bf16; the residual stream and logits fp32)."""
    H, I, V = cfg["hidden_size"], cfg["intermediate_size"], cfg["vocab_size"]
    nh, nkv, hd = cfg["num_attention_heads"], cfg["num_key_value_heads"], cfg["head_dim"]
    q, kv = nh * hd, nkv * hd
    keys = B * ((T // B) * context_before + (T // B) * (T // B + 1) / 2)      # query-key pairs under the causal mask
    cached = B * (context_before + T // B)                                    # tokens whose keys and values are read
    return {
        "embed": {"bytes": T * H * (2 + 4), "flops": 0},
        # per launch: how many norm kernels run depends on the step (products of very few or of many tokens fold them in)
        "norm": {"bytes": T * H * (4 + 2 + 4 + 2) + H * 4, "flops": 0, "per_launch": True},
        "qkv": {"bytes": layers * ((q + 2 * kv) * H * 2 + T * (H + q + 2 * kv) * 2), "flops": 2.0 * layers * T * H * (q + 2 * kv)},
        # per launch too: the step's one table of angles, then a kernel per layer unless the q/k/v product carries the
        # rotation in its epilogue (very few tokens, or a prompt portion)
        "rotary+write": {"bytes": T * (q + 2 * kv) * 2 * 2, "flops": 0, "per_launch": True, "first_launch_bytes": T * (hd * 4 + 4)},
        "attention": {"bytes": layers * (cached * 2 * kv * 2 + 2 * T * q * 2), "flops": 4.0 * layers * nh * hd * keys},
        "o": {"bytes": layers * (H * q * 2 + T * (q + H) * 2), "flops": 2.0 * layers * T * q * H},
        "gate_up": {"bytes": layers * (2 * I * H * 2 + T * (H + I) * 2), "flops": 4.0 * layers * T * H * I},
        "down": {"bytes": layers * (H * I * 2 + T * (I + H) * 2), "flops": 2.0 * layers * T * H * I},
        "head": {"bytes": V * H * 2 + logit_rows * (H * 2 + V * 4), "flops": 2.0 * logit_rows * H * V},
        "sampler": {"bytes": logit_rows * V * 4, "flops": 0},
    }


def kernel_table(totals: dict, work: dict, step_us: float, peaks: dict) -> dict:
    """The ``kernels`` block of one workload: per class its device microseconds (every kernel alone, one event
    between two launches), the bytes and flops it has to do, what it achieved, and the fraction of the measured
    peak that binds it: the copy bandwidth, or the cuBLAS burst figure (the right one for a kernel timed alone)
    where the flops are the larger share."""
    classes = {}
    for name, t in sorted(totals.items(), key=lambda kv: -kv[1]["us"]):
        w = work.get(name)
        row = {"us": round(t["us"], 1), "launches": t["launches"]}
        if w is not None and t["us"] > 0:
            if w.get("per_launch"):
                first = w.get("first_launch_bytes")
                n = t["launches"] if first is None else t["launches"] - 1
                w = {"bytes": w["bytes"] * n + (first or 0), "flops": w["flops"] * t["launches"]}
            # both yardsticks; the class is judged by the one that binds it (the larger fraction)
            gbs = w["bytes"] / (t["us"] * 1e-6) / 1e9
            tf = w["flops"] / (t["us"] * 1e-6) / 1e12
            f_mem, f_flop = gbs / peaks["hbm_gbs"], tf / peaks["bf16_tflops"]
            row.update(bytes=int(w["bytes"]), gbs=round(gbs, 1))
            if w["flops"]:
                row.update(flops=w["flops"], tflops=round(tf, 1))
            if f_flop > f_mem:
                row.update(frac=round(f_flop, 3), of="bf16_tflops")
            else:
                row.update(frac=round(f_mem, 3), of="hbm_gbs")
        classes[name] = row
    total = sum(t["us"] for t in totals.values())
    return {"step_us": round(step_us, 1), "sum_us": round(total, 1), "sum_over_step": round(total / step_us, 3) if step_us else None,
            "classes": classes}


def run_ours(args) -> dict:
    import numpy as np
    import torch

    from pyre_b200 import Engine, SamplingParams
    from pyre_b200.config import config_from_dict
    from pyre_b200.engine.step import StepEntry
    from pyre_b200.kernels import lib, ops

    peaks = load_peaks()
    cfg_raw = dict(CONFIG_7B)
    layers_full = cfg_raw["num_hidden_layers"]
    layers = args.layers or layers_full
    cfg_raw["num_hidden_layers"] = layers
    cfg = config_from_dict(cfg_raw)
    B = args.batch
    steps, warmup = args.steps, max(args.warmup, 3)
    biggest = max(B, 64 if not args.skip_points else B)
    tokens_needed = biggest * (PROMPT_LEN + 64 + SETTLE_STEPS + warmup + steps + PAGE_SIZE) + B * (2 * B + 64) + 2 * CONTEXT
    torch.cuda.set_device(0)
    engine = Engine(config=cfg, seed=0, dtype="bfloat16", device="cuda:0", page_size=PAGE_SIZE,
                    max_cache_tokens=tokens_needed, max_num_seqs=biggest, max_num_batched_tokens=PROMPT_LEN,
                    prefill_chunk=PROMPT_LEN, max_model_len=max(CONTEXT, PROMPT_LEN + SETTLE_STEPS + warmup + steps + 2 * B + 128))
    stepper, cache = engine.stepper, engine.cache
    vocab = cfg.vocab_size
    rng = np.random.default_rng(0)
    weight_bytes, kv_per_token, flops = model_numbers(cfg_raw, layers)
    clocks = ClockSampler(0)
    clocks.start()

    def ev():
        return torch.cuda.Event(enable_timing=True)

    # ---------------------------------------------------------------- prefill, 2,048 tokens in one step
    def prefill_once(rid):
        cache.begin(rid)
        ids = rng.integers(0, vocab, PROMPT_LEN).tolist()
        logits = stepper.step([StepEntry(rid, ids, [PROMPT_LEN - 1])])
        return ops.sample(logits)

    for i in range(2):
        prefill_once(("warm", i))
        cache.end(("warm", i))
    torch.cuda.synchronize()
    times = []
    for i in range(args.prefill_reps):
        a, b = ev(), ev()
        a.record()
        prefill_once(("pf", i))
        b.record()
        torch.cuda.synchronize()
        times.append(a.elapsed_time(b))
        cache.end(("pf", i))
    pf_ms = sorted(times)[len(times) // 2]
    pf_flops = flops(PROMPT_LEN, 0, 1)
    prefill = {"value": round(PROMPT_LEN / pf_ms * 1e3, 1), "tokens": PROMPT_LEN, "ms": round(pf_ms, 3),
               "frac": round(pf_flops / (pf_ms * 1e-3) / (peaks["bf16_tflops"] * 1e12), 4),
               # the same against the figure of a seconds-long loop under the power cap (this step repeats back to back)
               "frac_of_sustained": round(pf_flops / (pf_ms * 1e-3) / (peaks["bf16_tflops_sustained"] * 1e12), 4),
               "first_ms": round(times[0], 3)}

    # ---------------------------------------------------------------- decode, device-timed
    def decode_run(batch: int, n_warm: int, n_steps: int, tag: str):
        reqs = [(tag, i) for i in range(batch)]
        for r in reqs:
            cache.begin(r)
            stepper.step([StepEntry(r, rng.integers(0, vocab, PROMPT_LEN).tolist(), [])])
        n_warm += SETTLE_STEPS
        toks = rng.integers(0, vocab, (n_warm + n_steps, batch))

        def one(k):
            logits = stepper.step([StepEntry(r, [int(toks[k, i])], [0]) for i, r in enumerate(reqs)])
            return ops.sample(logits)

        for k in range(n_warm):
            one(k)
        torch.cuda.synchronize()
        launches0, mark0 = lib.launch_count, clocks.mark()
        a, b = ev(), ev()
        a.record()
        for k in range(n_warm, n_warm + n_steps):
            one(k)
        b.record()
        torch.cuda.synchronize()
        ms = a.elapsed_time(b) / n_steps
        info = {"ms": ms, "launches": lib.launch_count - launches0, "clock_rows": (mark0, clocks.mark()),
                "mean_context": PROMPT_LEN + n_warm + (n_steps + 1) / 2}
        for r in reqs:
            cache.end(r)
        return batch / ms * 1e3, info

    value, info = decode_run(B, warmup, steps, "dec")
    ms_per_step = info["ms"]
    step_bytes = weight_bytes + kv_per_token * info["mean_context"] * B
    achieved = step_bytes / (ms_per_step * 1e-3) / 1e9
    roofline = {"bound": "hbm", "achieved": round(achieved, 1), "peak": peaks["hbm_gbs"], "unit": "GB/s",
                "frac": round(achieved / peaks["hbm_gbs"], 4), "peak_source": peaks["source"]}
    clock_summary = clocks.summary(*info["clock_rows"])

    points = {}
    if not args.skip_points:
        for b_ in (1, 64):
            v, _ = decode_run(b_, 3, max(8, steps // 2), f"p{b_}")
            points[f"decode_b{b_}"] = round(v, 1)

    # ---------------------------------------------------------------- per kernel class, every kernel alone
    kernels = {}
    if not args.no_per_kernel:
        def timed(run_step, work):
            run_step()                                     # warm: the eager path's buffers and plans
            samples = []
            for _ in range(3):
                torch.cuda.synchronize()
                a, b = ev(), ev()
                with stepper.kernel_timing() as timer:
                    a.record()
                    run_step()
                    b.record()
                    totals = timer.totals()
                samples.append((a.elapsed_time(b) * 1e3, totals))
            samples.sort(key=lambda s_: s_[0])
            step_us, totals = samples[1]
            return kernel_table(totals, work, step_us, peaks)

        for b_ in ([1, 8, 64] if not args.skip_points else [B]):
            reqs = [("k", b_, i) for i in range(b_)]
            for r in reqs:
                cache.begin(r)
                stepper.step([StepEntry(r, rng.integers(0, vocab, PROMPT_LEN).tolist(), [])])
            kernels[f"decode_b{b_}"] = timed(
                lambda: ops.sample(stepper.step([StepEntry(r, [int(rng.integers(0, vocab))], [0]) for r in reqs])),
                class_work(cfg_raw, layers, b_, b_, PROMPT_LEN + 2, b_))
            for r in reqs:
                cache.end(r)
        serial = [0]

        def one_prefill():
            serial[0] += 1
            prefill_once(("kp", serial[0]))
            cache.end(("kp", serial[0]))
        kernels[f"prefill_{PROMPT_LEN}"] = timed(one_prefill, class_work(cfg_raw, layers, PROMPT_LEN, 1, 0, 1))

    # ---------------------------------------------------------------- end to end through Engine.step
    # every request must outlive the timed steps: the first one decodes while the others' prompts (cut to what the
    # token budget leaves beside the decoded tokens) are still being read, about B * PROMPT_LEN / (budget - B) steps
    sp = SamplingParams(max_new_tokens=SETTLE_STEPS + warmup + steps + 2 * B + 64, ignore_eos=True)
    sids = [engine.add_request(rng.integers(0, vocab, PROMPT_LEN).tolist(), params=sp) for _ in range(B)]
    live = [engine._requests[sid] for sid in sids]
    while any(not r.generated for r in live):
        engine.step()                      # the prompts, one per step under the token budget
    for _ in range(SETTLE_STEPS + warmup):
        engine.step()
    torch.cuda.synchronize()
    up0 = stepper._staging.bytes_uploaded + engine.sampler.bytes_uploaded
    down0 = engine.sampler.bytes_downloaded
    t0 = time.perf_counter()
    for _ in range(steps):
        engine.step()
    torch.cuda.synchronize()
    dt = time.perf_counter() - t0
    e2e = {"value": round(B * steps / dt, 1), "unit": "tokens/s",
           "h2d_bytes_per_step": (stepper._staging.bytes_uploaded + engine.sampler.bytes_uploaded - up0) // steps,
           "d2h_bytes_per_step": (engine.sampler.bytes_downloaded - down0) // steps}
    while engine.has_unfinished():
        engine.step()
    clocks.stop()
    stepper.check_device_errors()      # a kernel that gave up waiting would have raised the device's error word

    # ---------------------------------------------------------------- further sizes of the same architecture
    # decode tokens/s at longer contexts (this model) and at the 14B and 32B shapes (full layer counts, batch 8,
    # 2,048-token prompts): device-timed like `value`, each with its fraction of the copy roofline beside it
    if not args.skip_points and not args.skip_sizes:
        def decode_point(eng, cfg_raw_, n_layers, batch, context, n_warm=SETTLE_STEPS + 8, n_steps=24):
            st_, cache_ = eng.stepper, eng.cache
            wb, kvb, _ = model_numbers(cfg_raw_, n_layers)
            reqs = [("x", batch, context, i) for i in range(batch)]
            for r in reqs:
                cache_.begin(r)
                for lo in range(0, context, 8192):
                    st_.step([StepEntry(r, rng.integers(0, cfg_raw_["vocab_size"], min(8192, context - lo)).tolist(), [])])
            toks = rng.integers(0, cfg_raw_["vocab_size"], (n_warm + n_steps, batch))
            for k in range(n_warm):      # the clocks recover from the prefill's power cap meanwhile
                ops.sample(st_.step([StepEntry(r, [int(toks[k, i])], [0]) for i, r in enumerate(reqs)]))
            torch.cuda.synchronize()
            a, b = ev(), ev()
            a.record()
            for k in range(n_warm, n_warm + n_steps):
                ops.sample(st_.step([StepEntry(r, [int(toks[k, i])], [0]) for i, r in enumerate(reqs)]))
            b.record()
            torch.cuda.synchronize()
            ms = a.elapsed_time(b) / n_steps
            for r in reqs:
                cache_.end(r)
            frac = (wb + kvb * (context + n_warm + n_steps / 2) * batch) / (ms * 1e-3) / 1e9 / peaks["hbm_gbs"]
            return round(batch / ms * 1e3, 1), round(frac, 3)

        del stepper, cache, engine
        torch.cuda.empty_cache()
        long_cfg = dict(cfg_raw, max_position_embeddings=40960)
        eng = Engine(config=config_from_dict(long_cfg), seed=0, dtype="bfloat16", page_size=PAGE_SIZE, max_cache_tokens=8 * (32768 + SETTLE_STEPS + 256),
                     max_num_seqs=8, max_num_batched_tokens=8192, prefill_chunk=8192, max_model_len=40960)
        for batch, context in ((1, 8192), (1, 32768), (8, 8192), (8, 32768)):
            points[f"decode_b{batch}_ctx{context // 1024}k"], points[f"hbm_frac_b{batch}_ctx{context // 1024}k"] = \
                decode_point(eng, long_cfg, layers, batch, context)
        del eng
        torch.cuda.empty_cache()
        # many requests at the benchmark's context
        eng = Engine(config=cfg, seed=0, dtype="bfloat16", page_size=PAGE_SIZE, max_cache_tokens=256 * (PROMPT_LEN + SETTLE_STEPS + 64),
                     max_num_seqs=256, max_num_batched_tokens=PROMPT_LEN, prefill_chunk=PROMPT_LEN, max_model_len=CONTEXT)
        for batch in (128, 256):
            points[f"decode_b{batch}"], points[f"hbm_frac_b{batch}"] = decode_point(eng, cfg_raw, layers, batch, PROMPT_LEN, n_steps=16)
        del eng
        torch.cuda.empty_cache()
        if layers == layers_full:      # the other shapes only beside the full model
            for name in ("14b", "32b"):
                raw = dict(SHAPES[name])
                eng = Engine(config=config_from_dict(raw), seed=0, dtype="bfloat16", page_size=PAGE_SIZE, max_cache_tokens=8 * 2200 + 4096,
                             max_num_seqs=8, max_num_batched_tokens=2048, prefill_chunk=2048, max_model_len=4096)
                points[f"decode_b8_{name}"], points[f"hbm_frac_b8_{name}"] = decode_point(eng, raw, raw["num_hidden_layers"], 8, PROMPT_LEN)
                del eng
                torch.cuda.empty_cache()

    return {
        "metric": "decode tok/s (Qwen2.5-7B shape, batch 8, 2,048-token prompts)", "value": round(value, 1),
        "unit": "tokens/s", "n_gpus": 1, "steps": steps, "warmup": warmup, "untimed_steps": SETTLE_STEPS + warmup,
        "ms_per_step": round(ms_per_step, 4),
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
        "config": bench_config(cfg_raw, layers, layers_full, B),
        "clocks": clock_summary, "e2e": e2e, "gpu_launches": info["launches"], "prefill": prefill,
        "roofline": roofline, "points": points, "kernels": kernels, "impl": "ours",
    }


SHAPES = {
    # the two further workloads: continuous batching at the 14B shape, mixed steps at the 32B shape
    "14b": dict(architectures=["Qwen2ForCausalLM"], hidden_size=5120, intermediate_size=13824, num_hidden_layers=48,
                num_attention_heads=40, num_key_value_heads=8, head_dim=128, vocab_size=152064, rope_theta=1e6,
                rms_norm_eps=1e-5, tie_word_embeddings=False, max_position_embeddings=32768),
    "32b": dict(architectures=["Qwen2ForCausalLM"], hidden_size=5120, intermediate_size=27648, num_hidden_layers=64,
                num_attention_heads=40, num_key_value_heads=8, head_dim=128, vocab_size=152064, rope_theta=1e6,
                rms_norm_eps=1e-5, tie_word_embeddings=False, max_position_embeddings=32768),
}


def run_workload(args) -> dict:
    """The two other workloads of the baseline description, outside the one-line contract:
    ``serve14b``: continuous batching of 64 requests (prompts uniform in 128-4096 tokens, outputs
    uniform in 64-512) on the 14B shape through Engine.generate;
    ``mixed32b``: steps of 16 decoded tokens plus a 1,024-token prompt portion at contexts up
    to 8,192 on the 32B shape."""
    import numpy as np
    import torch

    from pyre_b200 import Engine, SamplingParams
    from pyre_b200.config import config_from_dict
    from pyre_b200.engine.step import StepEntry
    from pyre_b200.kernels import ops

    rng = np.random.default_rng(1)
    if args.workload == "serve14b":
        raw = dict(SHAPES["14b"])
        if args.layers:
            raw["num_hidden_layers"] = args.layers
        cfg = config_from_dict(raw)
        n_req = 64
        prompts = [rng.integers(0, cfg.vocab_size, int(rng.integers(128, 4097))).tolist() for _ in range(n_req)]
        outs_len = [int(rng.integers(64, 513)) for _ in range(n_req)]
        need = sum(len(p) + o for p, o in zip(prompts, outs_len))
        eng = Engine(config=cfg, seed=0, dtype="bfloat16", page_size=PAGE_SIZE, max_cache_tokens=int(need * args.cache_fraction),
                     max_num_seqs=64, max_num_batched_tokens=4096, prefill_chunk=2048, max_model_len=8192, record_steps=True)
        params = [SamplingParams(max_new_tokens=o, ignore_eos=True) for o in outs_len]
        eng.generate(prompts[:2], params[:2])       # warm-up: builds, graphs of small shapes
        torch.cuda.synchronize()
        eng.step_log.clear()
        t0 = time.perf_counter()
        res = eng.generate(prompts, params)
        torch.cuda.synchronize()
        dt = time.perf_counter() - t0
        st = eng.stats()
        eng.cache.check()
        n_out = sum(len(r.token_ids) for r in res)
        n_in = sum(len(p) for p in prompts)
        # the host's share: its own work per step against the time it spent waiting for the GPU.  Steps with prompt
        # tokens run kernel by kernel (hundreds of launches), decode-only steps replay a captured graph.
        log = eng.step_log
        mixed = [r for r in log if r["prompt_tokens"]]
        host = {"steps": len(log), "steps_with_prompt_tokens": len(mixed),
                "host_ms_total": round(sum(r["host_ms"] for r in log), 1), "wait_ms_total": round(sum(r["wait_ms"] for r in log), 1),
                "host_ms_per_prompt_step": round(sum(r["host_ms"] for r in mixed) / max(1, len(mixed)), 3),
                "host_ms_per_decode_step": round(sum(r["host_ms"] for r in log if not r["prompt_tokens"]) / max(1, len(log) - len(mixed)), 3),
                "steps_the_host_did_not_wait_in": sum(1 for r in log if r["wait_ms"] < 0.05)}
        return {"workload": "serve14b", "layers": cfg.num_hidden_layers, "requests": n_req, "prompt_tokens": n_in,
                "output_tokens": n_out, "seconds": round(dt, 3), "output_tok_s": round(n_out / dt, 1),
                "total_tok_s": round((n_in + n_out) / dt, 1), "steps": st["steps"], "preempted": st["preempted"],
                "cache_tokens": int(need * args.cache_fraction), "finished": sum(r.finish_reason == "length" for r in res),
                "graph_captures": eng.stepper.graph_captures, "graph_replays": eng.stepper.graph_replays,
                "capture_seconds": round(eng.stepper.capture_seconds, 3), "host": host}
    raw = dict(SHAPES["32b"])
    if args.layers:
        raw["num_hidden_layers"] = args.layers
    cfg = config_from_dict(raw)
    n_dec, chunk, ctx = 16, 1024, 8192
    eng = Engine(config=cfg, seed=0, dtype="bfloat16", page_size=PAGE_SIZE, max_cache_tokens=(n_dec + 1) * (ctx + 64),
                 max_num_seqs=n_dec + 1, max_num_batched_tokens=4096, prefill_chunk=4096, max_model_len=ctx + 64)
    st, cache = eng.stepper, eng.cache
    reqs = list(range(n_dec))
    for r in reqs:                              # decoding requests at contexts between 2,048 and 8,000
        cache.begin(r)
        n = int(rng.integers(2048, ctx - 200))
        for lo in range(0, n, 4096):
            st.step([StepEntry(r, rng.integers(0, cfg.vocab_size, min(4096, n - lo)).tolist(), [])])
    cache.begin("p")
    times = []
    for k in range(ctx // chunk - 1):           # the prompt grows by 1,024 tokens per step beside 16 decoded tokens
        entries = [StepEntry(r, [int(rng.integers(0, cfg.vocab_size))], [0]) for r in reqs]
        entries.append(StepEntry("p", rng.integers(0, cfg.vocab_size, chunk).tolist(), [chunk - 1]))
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        ops.sample(st.step(entries))
        b.record()
        torch.cuda.synchronize()
        times.append(a.elapsed_time(b))
    cache.check()
    ms = sorted(times[1:])[len(times[1:]) // 2]
    return {"workload": "mixed32b", "layers": cfg.num_hidden_layers, "tokens_per_step": n_dec + chunk,
            "ms_per_step_median": round(ms, 2), "tok_s": round((n_dec + chunk) / ms * 1e3, 1),
            "ms_first_last": [round(times[1], 2), round(times[-1], 2)]}


def run_modovik(args) -> dict:
    """``--workload modovik``: the Modovik design at layer sizes of the 7B shape (random weights) beside the Qwen2.5
    decoder at equal sizes and as many layers: a 2,048-token prompt step and decode steps at batch 8 and 64 with
    2,048 tokens of context, device-timed, and per kernel class the device time of one such step with the
    fraction of the measured peak (copy bandwidth, or the cuBLAS figure where the flops bind).  Four layers:
    attention, lightning, attention, an attention layer that reads the third layer's cache."""
    import numpy as np
    import torch

    from pyre_b200 import Engine
    from pyre_b200.config import config_from_dict
    from pyre_b200.engine.step import StepEntry
    from pyre_b200.kernels import ops

    peaks = load_peaks()
    H, I, nh, nkv, hd, V = 3584, 18944, 28, 4, 128, 32768
    rot = {"dims": 64, "base": 1e6}
    att = lambda **kw: {"type": "attention", "mixer": dict(heads=nh, kv_heads=nkv, dim=hd, vdim=hd, scale=hd ** -0.5, rot=rot, **kw),
                        "mlp": {"kind": "dense", "ff": I}}
    raw_m = {"architecture": "Modovik", "vocab": V, "width": H, "norm": {"eps": 1e-6}, "layers": [
        att(), {"type": "lightning", "mixer": {"heads": nh, "dim": hd, "vdim": hd, "decay": [1.0 - 2.0 ** (-5 - 3 * i / nh) for i in range(nh)]},
                "mlp": {"kind": "dense", "ff": I}}, att(), att(kv_from=2)]}
    L = len(raw_m["layers"])
    raw_q = dict(CONFIG_7B, num_hidden_layers=L, vocab_size=V)
    T, ctx_len, reps = PROMPT_LEN, 2048, max(3, args.prefill_reps)
    rng = np.random.default_rng(0)
    q, kv = nh * hd, nkv * hd

    def work_modovik(Tn, B, before):
        """bytes and flops per class of one step of the four layers (three attention layers, one of them without
        keys and values of its own; one lightning layer)"""
        keys = B * ((Tn // B) * before + (Tn // B) * (Tn // B + 1) / 2)
        cached = B * (before + Tn // B)
        proj_att = 2 * (2 * q + 2 * kv) + (2 * q)          # columns of the stacked projections: q k v g, q k v g, q g
        proj_lin = 4 * q
        return {
            "qkv": {"bytes": (proj_att + proj_lin) * H * 2 + Tn * (L * H + proj_att + proj_lin) * 2, "flops": 2.0 * Tn * H * (proj_att + proj_lin)},
            "attention": {"bytes": 3 * (cached * 2 * kv * 2 + 2 * Tn * q * 2), "flops": 4.0 * 3 * nh * hd * keys},
            "linear_attention": {"bytes": Tn * 3 * q * 2 + Tn * q * 4 + B * 2 * nh * hd * hd * 4, "flops": 4.0 * Tn * nh * hd * hd},
            "o": {"bytes": L * (H * q * 2 + Tn * (q + H) * 2), "flops": 2.0 * L * Tn * q * H},
            "up": {"bytes": L * (I * H * 2 + Tn * (H + I) * 2), "flops": 2.0 * L * Tn * H * I},
            "down": {"bytes": L * (H * I * 2 + Tn * (I + H) * 2), "flops": 2.0 * L * Tn * H * I},
            "activation": {"bytes": L * Tn * I * 4, "flops": 0},
            "norm": {"bytes": Tn * H * (2 + 4 + 4 + 2), "flops": 0, "per_launch": True},
            "gate": {"bytes": Tn * q * (2 + 2 + 2), "flops": 0, "per_launch": True},
            "rotary+write": {"bytes": Tn * (q + 2 * kv) * 2 * 2, "flops": 0, "per_launch": True},
            "head": {"bytes": V * H * 2 + B * (H * 2 + V * 4), "flops": 2.0 * B * H * V},
            "embed": {"bytes": Tn * H * (2 + 4), "flops": 0},
        }

    out = {"workload": "modovik", "layers": L, "peaks": peaks, "sizes": {"width": H, "ff": I, "heads": nh, "kv_heads": nkv,
           "dim": hd, "vdim": hd, "vocab": V, "prompt": T, "decode_context": ctx_len}, "models": {}}
    for name, raw in (("modovik", raw_m), ("qwen2", raw_q)):
        cfg = config_from_dict(raw)
        biggest = 64
        eng = Engine(config=cfg, seed=0, dtype="bfloat16", device="cuda:0", page_size=PAGE_SIZE,
                     max_cache_tokens=biggest * (ctx_len + 256) + 4 * T, max_num_seqs=biggest + 1, max_num_batched_tokens=T,
                     prefill_chunk=T, max_model_len=ctx_len + 256)
        st, cache = eng.stepper, eng.cache

        def ev():
            return torch.cuda.Event(enable_timing=True)

        def prompt(rid, n=T):
            cache.begin(rid)
            return st.step([StepEntry(rid, rng.integers(0, V, n).tolist(), [n - 1])])

        for i in range(2):
            prompt(("warm", i))
            cache.end(("warm", i))
        times = []
        for i in range(reps):
            a, b = ev(), ev()
            a.record()
            prompt(("pf", i))
            b.record()
            torch.cuda.synchronize()
            times.append(a.elapsed_time(b))
            cache.end(("pf", i))
        res = {"prefill_ms": round(sorted(times)[len(times) // 2], 3)}
        res["prefill_tok_s"] = round(T / res["prefill_ms"] * 1e3, 1)
        with st.kernel_timing() as timer:
            prompt("timed")
        cache.end("timed")
        work = work_modovik(T, 1, 0) if name == "modovik" else class_work(raw_q, L, T, 1, 0, 1)
        res["prefill_kernels"] = kernel_table(timer.totals(), work, res["prefill_ms"] * 1e3, peaks)
        for i in range(biggest):
            prompt(("d", i), ctx_len)
        for B in (8, 64):
            reqs = [("d", i) for i in range(B)]
            step = lambda: st.step([StepEntry(r, [int(rng.integers(0, V))], [0]) for r in reqs])
            for _ in range(max(4, args.warmup)):
                step()
            torch.cuda.synchronize()
            n = min(args.steps, 32)
            a, b = ev(), ev()
            a.record()
            for _ in range(n):
                step()
            b.record()
            torch.cuda.synchronize()
            ms = a.elapsed_time(b) / n
            res[f"decode_b{B}_ms"] = round(ms, 4)
            res[f"decode_b{B}_tok_s"] = round(B / ms * 1e3, 1)
            with st.kernel_timing() as timer:
                step()
            work = work_modovik(B, B, ctx_len + 40) if name == "modovik" else class_work(raw_q, L, B, B, ctx_len + 40, B)
            res[f"decode_b{B}_kernels"] = kernel_table(timer.totals(), work, ms * 1e3, peaks)
        out["models"][name] = res
        del eng, st, cache
        torch.cuda.empty_cache()
    return out


def run_pivinex(args) -> dict:
    """``--workload pivinex``: the Pivinex design (latent attention, a gated gelu and a routed feed-forward, random
    weights) at two sets of layer sizes beside the Qwen2.5 decoder at equal width, heads and feed-forward size and as
    many layers: a 2,048-token prompt step and decode steps at batch 8 and 64 with 2,048 tokens of context,
    device-timed, and per kernel class the device time of one such step with the fraction of the measured peak
    (copy bandwidth, or the cuBLAS figure where the flops bind).  Two layers: a dense and a routed feed-forward."""
    import numpy as np
    import torch

    from pyre_b200 import Engine
    from pyre_b200.config import config_from_dict
    from pyre_b200.engine.step import StepEntry

    peaks = load_peaks()
    V = 32768
    sizes = {
        # width, heads, dim, rot, vdim, q_rank, kv_rank, window, dense ff, experts, identity, top, expert ff
        "2k": dict(H=2048, nh=16, dn=128, dr=64, dv=128, qr=768, kr=256, win=1024, I=8192, E=32, ident=2, top=4, ff=1024),
        "3.5k": dict(H=3584, nh=28, dn=128, dr=64, dv=128, qr=1536, kr=512, win=4096, I=18944, E=64, ident=0, top=6, ff=1408),
    }
    T, ctx_len, reps = PROMPT_LEN, 2048, max(3, args.prefill_reps)
    rng = np.random.default_rng(0)
    out = {"workload": "pivinex", "layers": 2, "peaks": peaks, "prompt": T, "decode_context": ctx_len, "sizes": {}}
    for tag, z in sizes.items():
        H, nh, dn, dr, dv, qr, kr, win, I, E, ident, top, ff = (z[k] for k in ("H", "nh", "dn", "dr", "dv", "qr", "kr", "win", "I", "E", "ident", "top", "ff"))
        mixer = {"heads": nh, "dim": dn, "rot_dim": dr, "vdim": dv, "q_rank": qr, "kv_rank": kr, "scale": (dn + dr) ** -0.5,
                 "mask": {"size": win}, "rot": {"dims": dr, "base": 1e6}}
        raw_p = {"architecture": "Pivinex", "vocab": V, "width": H, "norm": {"eps": 1e-6}, "residual_mult": 0.5, "layers": [
            {"type": "latent_attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": I}},
            {"type": "latent_attention", "mixer": mixer, "mlp": {"kind": "moe", "expert": {"ff": ff},
                                                                "router": {"experts": E, "identity": ident, "top": top, "scale": 1.0}}}]}
        L = 2
        raw_q = dict(CONFIG_7B, hidden_size=H, intermediate_size=I, num_attention_heads=nh, num_key_value_heads=4, head_dim=128,
                     num_hidden_layers=L, vocab_size=V)
        row = -(-(kr + dr) // 16) * 16

        def work_pivinex(Tn, B, before):
            """bytes and flops per class of one step of the two layers"""
            per = Tn // B
            first = np.arange(before, before + per)                      # positions of an entry's tokens
            keys = B * float(np.minimum(first + 1, win).sum())           # query-key pairs inside the window
            cached = B * min(before + per, win + per)                    # cached rows that are read
            pairs = Tn * top                                             # (token, expert) pairs, all with weights at most
            used = min(E, pairs)                                         # experts whose weights are read
            down_cols = qr + kr + dr
            return {
                "qkv": {"bytes": L * (down_cols * H * 2 + Tn * (H + down_cols) * 2), "flops": 2.0 * L * Tn * H * down_cols},
                "q_up": {"bytes": L * (nh * (dn + dr) * qr * 2 + Tn * (qr + nh * (dn + dr)) * 2), "flops": 2.0 * L * Tn * qr * nh * (dn + dr)},
                "absorb": {"bytes": L * (nh * dn * kr * 2 + Tn * nh * (dn + kr) * 2), "flops": 2.0 * L * Tn * nh * dn * kr},
                "latent_attention": {"bytes": L * (cached * row * 2 + Tn * nh * (row + kr) * 2), "flops": 2.0 * L * nh * (kr + dr + kr) * keys},
                "v_up": {"bytes": L * (nh * dv * kr * 2 + Tn * nh * (kr + dv) * 2), "flops": 2.0 * L * Tn * nh * kr * dv},
                "o": {"bytes": L * (H * nh * dv * 2 + Tn * (nh * dv + H) * 2), "flops": 2.0 * L * Tn * nh * dv * H},
                "gate_up": {"bytes": 2 * I * H * 2 + Tn * (H + 2 * I) * 2 + Tn * 3 * I * 2, "flops": 4.0 * Tn * H * I},
                "down": {"bytes": H * I * 2 + Tn * (I + H) * 2, "flops": 2.0 * Tn * H * I},
                "experts_gate_up": {"bytes": used * 2 * ff * H * 2 + pairs * (H + 2 * ff) * 2, "flops": 4.0 * pairs * H * ff},
                "experts_down": {"bytes": used * H * ff * 2 + pairs * (ff * 2 + H * 4), "flops": 2.0 * pairs * H * ff},
                "router": {"bytes": (E + ident) * H * 4 + Tn * H * 2 + pairs * H * 4 + Tn * H * 4, "flops": 2.0 * Tn * H * (E + ident)},
                "activation": {"bytes": pairs * 3 * ff * 2, "flops": 0},
                "norm": {"bytes": Tn * H * (2 + 2 + 4 + 4 + 2), "flops": 0, "per_launch": True},
                "rotary+write": {"bytes": Tn * (down_cols + qr + row) * 2, "flops": 0, "per_launch": True},
                "head": {"bytes": V * H * 2 + B * (H * 2 + V * 4), "flops": 2.0 * B * H * V},
                "embed": {"bytes": Tn * H * (2 + 4), "flops": 0},
            }

        block = {"sizes": z, "models": {}}
        for name, raw in (("pivinex", raw_p), ("qwen2", raw_q)):
            cfg = config_from_dict(raw)
            biggest = 64
            eng = Engine(config=cfg, seed=0, dtype="bfloat16", device="cuda:0", page_size=PAGE_SIZE,
                         max_cache_tokens=biggest * (ctx_len + 256) + 4 * T, max_num_seqs=biggest + 1, max_num_batched_tokens=T,
                         prefill_chunk=T, max_model_len=ctx_len + 256)
            st, cache = eng.stepper, eng.cache

            def ev():
                return torch.cuda.Event(enable_timing=True)

            def prompt(rid, n=T):
                cache.begin(rid)
                return st.step([StepEntry(rid, rng.integers(0, V, n).tolist(), [n - 1])])

            for i in range(2):
                prompt(("warm", i))
                cache.end(("warm", i))
            times = []
            for i in range(reps):
                a, b = ev(), ev()
                a.record()
                prompt(("pf", i))
                b.record()
                torch.cuda.synchronize()
                times.append(a.elapsed_time(b))
                cache.end(("pf", i))
            res = {"prefill_ms": round(sorted(times)[len(times) // 2], 3)}
            res["prefill_tok_s"] = round(T / res["prefill_ms"] * 1e3, 1)
            with st.kernel_timing() as timer:
                prompt("timed")
            cache.end("timed")
            work = work_pivinex(T, 1, 0) if name == "pivinex" else class_work(raw_q, L, T, 1, 0, 1)
            res["prefill_kernels"] = kernel_table(timer.totals(), work, res["prefill_ms"] * 1e3, peaks)
            for i in range(biggest):
                prompt(("d", i), ctx_len)
            for B in (8, 64):
                reqs = [("d", i) for i in range(B)]
                step = lambda: st.step([StepEntry(r, [int(rng.integers(0, V))], [0]) for r in reqs])
                for _ in range(max(4, args.warmup)):
                    step()
                torch.cuda.synchronize()
                n = min(args.steps, 32)
                a, b = ev(), ev()
                a.record()
                for _ in range(n):
                    step()
                b.record()
                torch.cuda.synchronize()
                ms = a.elapsed_time(b) / n
                res[f"decode_b{B}_ms"] = round(ms, 4)
                res[f"decode_b{B}_tok_s"] = round(B / ms * 1e3, 1)
                with st.kernel_timing() as timer:
                    step()
                work = work_pivinex(B, B, ctx_len + 40) if name == "pivinex" else class_work(raw_q, L, B, B, ctx_len + 40, B)
                res[f"decode_b{B}_kernels"] = kernel_table(timer.totals(), work, ms * 1e3, peaks)
            block["models"][name] = res
            del eng, st, cache
            torch.cuda.empty_cache()
        out["sizes"][tag] = block
    return out


def _measure_design(cfg, work, args, peaks, V, T, ctx_len, rng, batches=(8, 64)) -> dict:
    """One engine with random weights of ``cfg``: the device time of a ``T``-token prompt step (median of a few) and of
    decode steps at the given batch sizes with ``ctx_len`` tokens of context, each with its per-class table;
    ``work(tokens, entries, context_before)`` gives the classes' bytes and flops."""
    import torch

    from pyre_b200 import Engine
    from pyre_b200.engine.step import StepEntry

    biggest, reps = max(batches), max(3, args.prefill_reps)
    eng = Engine(config=cfg, seed=0, dtype="bfloat16", device="cuda:0", page_size=PAGE_SIZE,
                 max_cache_tokens=biggest * (ctx_len + 256) + 4 * T, max_num_seqs=biggest + 1, max_num_batched_tokens=T,
                 prefill_chunk=T, max_model_len=ctx_len + 256)
    st, cache = eng.stepper, eng.cache

    def ev():
        return torch.cuda.Event(enable_timing=True)

    def prompt(rid, n=T):
        cache.begin(rid)
        return st.step([StepEntry(rid, rng.integers(0, V, n).tolist(), [n - 1])])

    for i in range(2):
        prompt(("warm", i))
        cache.end(("warm", i))
    times = []
    for i in range(reps):
        a, b = ev(), ev()
        a.record()
        prompt(("pf", i))
        b.record()
        torch.cuda.synchronize()
        times.append(a.elapsed_time(b))
        cache.end(("pf", i))
    res = {"prefill_ms": round(sorted(times)[len(times) // 2], 3)}
    res["prefill_tok_s"] = round(T / res["prefill_ms"] * 1e3, 1)

    def timed(run):
        """Per-class times of the least disturbed of three steps (a stall of the host between two launches shows as a class's time)."""
        best = None
        for _ in range(3):
            with st.kernel_timing() as timer:
                run()
            totals = timer.totals()
            if best is None or sum(t["us"] for t in totals.values()) < sum(t["us"] for t in best.values()):
                best = totals
        return best

    def timed_prompt():
        prompt("timed")
        cache.end("timed")
    res["prefill_kernels"] = kernel_table(timed(timed_prompt), work(T, 1, 0), res["prefill_ms"] * 1e3, peaks)
    for i in range(biggest):
        prompt(("d", i), ctx_len)
    for B in batches:
        reqs = [("d", i) for i in range(B)]
        step = lambda: st.step([StepEntry(r, [int(rng.integers(0, V))], [0]) for r in reqs])
        for _ in range(max(4, args.warmup)):
            step()
        torch.cuda.synchronize()
        n = min(args.steps, 32)
        a, b = ev(), ev()
        a.record()
        for _ in range(n):
            step()
        b.record()
        torch.cuda.synchronize()
        ms = a.elapsed_time(b) / n
        res[f"decode_b{B}_ms"] = round(ms, 4)
        res[f"decode_b{B}_tok_s"] = round(B / ms * 1e3, 1)
        res[f"decode_b{B}_kernels"] = kernel_table(timed(step), work(B, B, ctx_len + 40), ms * 1e3, peaks)
    del eng, st, cache
    torch.cuda.empty_cache()
    return res


def run_tekarax(args) -> dict:
    """``--workload tekarax``: the Tekarax design (random weights) at two sets of layer sizes, three layers (a
    recurrent one with a dense feed-forward, a windowed latent-attention one with routed experts, a softmax-attention
    one with a dense feed-forward), beside the package's closest layers at equal sizes: Modovik's constant-decay
    recurrent layer and its attention layer with dense feed-forwards, and Pivinex's latent-attention layer with routed
    experts.  A 2,048-token prompt step and decode steps at batch 8 and 64 with 2,048 tokens of context, device-timed,
    and per kernel class the device time of one such step with the fraction of the measured peak."""
    import numpy as np

    from pyre_b200.config import config_from_dict

    peaks = load_peaks()
    V = 32768
    sizes = {
        # width, attention heads / kv heads / dim, recurrent head size and decay map, latent rank and window, feed-forwards
        "2k": dict(H=2048, nh=16, nkv=4, hd=128, wd=64, wr=64, kr=320, win=1024, I=8192, E=32, top=4, ff=1024, sh=2048),
        "3.5k": dict(H=3584, nh=28, nkv=4, hd=128, wd=64, wr=96, kr=512, win=4096, I=18944, E=64, top=6, ff=1408, sh=2816),
    }
    T, ctx_len = PROMPT_LEN, 2048
    rng = np.random.default_rng(0)
    out = {"workload": "tekarax", "peaks": peaks, "prompt": T, "decode_context": ctx_len, "sizes": {}}
    for tag, z in sizes.items():
        H, nh, nkv, hd, wd, wr, kr, win, I, E, top, ff, sh = (z[k] for k in ("H", "nh", "nkv", "hd", "wd", "wr", "kr", "win", "I", "E", "top", "ff", "sh"))
        wh = H // wd                                           # recurrent heads: heads x size = width
        q, kv, row = nh * hd, nkv * hd, -(-kr // 16) * 16
        rot = {"dims": 64, "base": 1e6, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}
        moe = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": E, "top": top}, "shared": {"ff": sh}}
        raw_t = {"architecture": "Tekarax", "vocab": V, "width": H, "norm": {"eps": 1e-6}, "layers": [
            {"type": "wkv", "mixer": {"heads": wh, "dim": wd, "decay_rank": wr}, "mlp": {"kind": "dense", "ff": I}},
            {"type": "latent_attention", "mixer": {"heads": nh, "dim": hd, "vdim": hd, "kv_rank": kr, "scale": hd ** -0.5, "mask": {"size": win}}, "mlp": moe},
            {"type": "attention", "mixer": {"heads": nh, "kv_heads": nkv, "dim": hd, "vdim": hd, "scale": hd ** -0.5, "rot": rot},
             "mlp": {"kind": "dense", "ff": I}}]}
        raw_m = {"architecture": "Modovik", "vocab": V, "width": H, "norm": {"eps": 1e-6}, "layers": [
            {"type": "lightning", "mixer": {"heads": wh, "dim": wd, "vdim": wd, "decay": [1.0 - 2.0 ** (-5 - 3 * i / wh) for i in range(wh)]},
             "mlp": {"kind": "dense", "ff": I}},
            {"type": "attention", "mixer": dict(heads=nh, kv_heads=nkv, dim=hd, vdim=hd, scale=hd ** -0.5, rot={"dims": 64, "base": 1e6}),
             "mlp": {"kind": "dense", "ff": I}}]}
        pr = min(64, kr // 4)                                  # Pivinex rotates a part of each row: rank + part = the same row size
        raw_p = {"architecture": "Pivinex", "vocab": V, "width": H, "norm": {"eps": 1e-6}, "residual_mult": 0.5, "layers": [
            {"type": "latent_attention", "mixer": {"heads": nh, "dim": hd, "rot_dim": pr, "vdim": hd, "q_rank": 768, "kv_rank": kr - pr,
                                                   "scale": (hd + pr) ** -0.5, "mask": {"size": win}, "rot": {"dims": pr, "base": 1e6}},
             "mlp": {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": E, "identity": 0, "top": top, "scale": 1.0}}}]}
        whd = wh * wd

        def attention_pairs(Tn, B, before, window=None):
            first = np.arange(before, before + Tn // B)
            return B * float((np.minimum(first + 1, window) if window else first + 1).sum())

        def dense(Tn, n):
            return {"up": {"bytes": n * (I * H * 2 + Tn * (H + I) * 2), "flops": 2.0 * n * Tn * H * I},
                    "down": {"bytes": n * (H * I * 2 + Tn * (I + H) * 2), "flops": 2.0 * n * Tn * H * I}}

        def routed(Tn, shared):
            pairs = Tn * top
            used = min(E, pairs)
            return {"experts_gate_up": {"bytes": used * 2 * ff * H * 2 + pairs * (H + 2 * ff) * 2, "flops": 4.0 * pairs * H * ff},
                    "experts_down": {"bytes": used * H * ff * 2 + pairs * (ff * 2 + H * 4), "flops": 2.0 * pairs * H * ff},
                    "router": {"bytes": E * H * 4 + Tn * H * 2 + pairs * H * (4 + 2) + Tn * H * 4, "flops": 2.0 * Tn * H * E},
                    **({"gate_up": {"bytes": 2 * shared * H * 2 + Tn * (H + 2 * shared) * 2, "flops": 4.0 * Tn * H * shared}} if shared else {})}

        def tail(Tn, B):
            return {"head": {"bytes": V * H * 2 + B * (H * 2 + V * 4), "flops": 2.0 * B * H * V}, "embed": {"bytes": Tn * H * (2 + 4), "flops": 0}}

        def work_tekarax(Tn, B, before):
            proj = 4 * whd + (q + 2 * kv + nh) + kr            # r k v g | q k v gates | latent
            cached_l = B * min(before + Tn // B, win + Tn // B)
            cached_a = B * (before + Tn // B)
            w = {
                "qkv": {"bytes": proj * H * 2 + Tn * (6 * H + proj) * 2, "flops": 2.0 * Tn * H * proj},
                "decay": {"bytes": (wr * H + whd * wr) * 2 + Tn * (H + 2 * wr) * 2 + Tn * whd * 4, "flops": 2.0 * Tn * wr * (H + whd)},
                "recurrence": {"bytes": Tn * (H * 2 * 6 + whd * (2 * 5 + 4)) + B * (2 * wh * wd * wd + 2 * H) * 4, "flops": 6.0 * Tn * wh * wd * wd},
                "q_up": {"bytes": q * H * 2 + Tn * (H + q) * 2, "flops": 2.0 * Tn * H * q},
                "absorb": {"bytes": nh * hd * kr * 2 + Tn * nh * (hd + row) * 2, "flops": 2.0 * Tn * nh * hd * kr},
                "v_up": {"bytes": nh * hd * kr * 2 + Tn * nh * (kr + hd) * 2, "flops": 2.0 * Tn * nh * kr * hd},
                "latent_attention": {"bytes": cached_l * row * 2 + Tn * nh * (row + kr) * 2, "flops": 4.0 * nh * kr * attention_pairs(Tn, B, before, win)},
                "attention": {"bytes": cached_a * 2 * kv * 2 + 2 * Tn * q * 2, "flops": 4.0 * nh * hd * attention_pairs(Tn, B, before)},
                "o": {"bytes": (whd + 2 * q) * H * 2 + Tn * (whd + 2 * q + 3 * H) * 2, "flops": 2.0 * Tn * H * (whd + 2 * q)},
                "residual_gate": {"bytes": 6 * (H * H * 2 + Tn * 2 * H * 2), "flops": 2.0 * 6 * Tn * H * H},
                "activation": {"bytes": 2 * Tn * I * 4 + Tn * top * 3 * ff * 2 + Tn * 3 * sh * 2 + Tn * wr * 4, "flops": 0},
                "norm": {"bytes": Tn * H * (2 + 2 + 4 + 4), "flops": 0, "per_launch": True},
                "gate": {"bytes": Tn * q * (2 + 2), "flops": 0, "per_launch": True},
                "rotary+write": {"bytes": Tn * (q + 2 * kv) * 2 * 2, "flops": 0, "per_launch": True},
                **dense(Tn, 2), **routed(Tn, sh), **tail(Tn, B)}
            return w

        def work_modovik(Tn, B, before):
            proj = 4 * whd + (2 * q + 2 * kv)
            return {
                "qkv": {"bytes": proj * H * 2 + Tn * (2 * H + proj) * 2, "flops": 2.0 * Tn * H * proj},
                "attention": {"bytes": B * (before + Tn // B) * 2 * kv * 2 + 2 * Tn * q * 2, "flops": 4.0 * nh * hd * attention_pairs(Tn, B, before)},
                "linear_attention": {"bytes": Tn * 3 * whd * 2 + Tn * whd * 4 + B * 2 * wh * wd * wd * 4, "flops": 4.0 * Tn * wh * wd * wd},
                "o": {"bytes": (whd + q) * H * 2 + Tn * (whd + q + 2 * H) * 2, "flops": 2.0 * Tn * H * (whd + q)},
                "activation": {"bytes": 2 * Tn * I * 4, "flops": 0},
                "norm": {"bytes": Tn * H * (2 + 4 + 4 + 2), "flops": 0, "per_launch": True},
                "gate": {"bytes": Tn * q * (2 + 2 + 2), "flops": 0, "per_launch": True},
                "rotary+write": {"bytes": Tn * (q + 2 * kv) * 2 * 2, "flops": 0, "per_launch": True},
                **dense(Tn, 2), **tail(Tn, B)}

        def work_pivinex(Tn, B, before):
            down_cols = 768 + kr
            cached = B * min(before + Tn // B, win + Tn // B)
            return {
                "qkv": {"bytes": down_cols * H * 2 + Tn * (H + down_cols) * 2, "flops": 2.0 * Tn * H * down_cols},
                "q_up": {"bytes": nh * (hd + pr) * 768 * 2 + Tn * (768 + nh * (hd + pr)) * 2, "flops": 2.0 * Tn * 768 * nh * (hd + pr)},
                "absorb": {"bytes": nh * hd * (kr - pr) * 2 + Tn * nh * (hd + kr) * 2, "flops": 2.0 * Tn * nh * hd * (kr - pr)},
                "latent_attention": {"bytes": cached * row * 2 + Tn * nh * (row + kr) * 2, "flops": 2.0 * nh * (2 * kr - pr) * attention_pairs(Tn, B, before, win)},
                "v_up": {"bytes": nh * hd * (kr - pr) * 2 + Tn * nh * (kr + hd) * 2, "flops": 2.0 * Tn * nh * (kr - pr) * hd},
                "o": {"bytes": H * q * 2 + Tn * (q + H) * 2, "flops": 2.0 * Tn * q * H},
                "activation": {"bytes": Tn * top * 3 * ff * 2, "flops": 0},
                "norm": {"bytes": Tn * H * (2 + 2 + 4 + 4 + 2), "flops": 0, "per_launch": True},
                "rotary+write": {"bytes": Tn * (down_cols + 768 + row) * 2, "flops": 0, "per_launch": True},
                **routed(Tn, 0), **tail(Tn, B)}

        block = {"sizes": dict(z, recurrent_heads=wh), "models": {}}
        for name, raw, work in (("tekarax", raw_t, work_tekarax), ("modovik", raw_m, work_modovik), ("pivinex", raw_p, work_pivinex)):
            block["models"][name] = dict(layers=len(raw["layers"]), **_measure_design(config_from_dict(raw), work, args, peaks, V, T, ctx_len, rng))
        out["sizes"][tag] = block
    return out


def run_nipudra(args) -> dict:
    """``--workload nipudra``: the Nipudra design (random weights) at two sets of layer sizes, three layers (retention,
    differential attention over a window with short convolutions, a state-space recurrence; each with routed experts
    and a shared one, and a per-layer input from a side table), beside the package's closest layers at equal sizes:
    two Tekarax layers (its recurrent layer and its softmax-attention layer, each with routed experts and a shared
    one between two layer norms per sublayer) and Modovik's constant-decay recurrent layer with a dense feed-forward.
    A 2,048-token prompt step and decode steps at batch 8 and 64 with 2,048 tokens of context, device-timed, and per
    kernel class the device time of one such step with the fraction of the measured peak."""
    import numpy as np

    from pyre_b200.config import config_from_dict

    peaks = load_peaks()
    V = 32768
    sizes = {
        # width; heads / key-value heads / map size of the attention; retention heads of 128; state-space heads of 64
        # with a state of 128 rows in 8 groups; window; experts, chosen, their size, the shared one's; side table
        "2k": dict(H=2048, nh=8, nkv=2, hd=128, win=1024, E=32, top=4, ff=1024, sh=2048, side=256),
        "3.5k": dict(H=3584, nh=14, nkv=2, hd=128, win=4096, E=64, top=6, ff=1408, sh=2816, side=256),
    }
    T, ctx_len = PROMPT_LEN, 2048
    rng = np.random.default_rng(0)
    out = {"workload": "nipudra", "peaks": peaks, "prompt": T, "decode_context": ctx_len, "sizes": {}}
    for tag, z in sizes.items():
        H, nh, nkv, hd, win, E, top, ff, sh, side = (z[k] for k in ("H", "nh", "nkv", "hd", "win", "E", "top", "ff", "sh", "side"))
        rh, rd = H // 128, 128                                 # retention: heads x size = width
        mh, P, N, G, taps = 2 * H // 64, 64, 128, 8, 4         # state space: inner = 2 x width
        inner, conv_ch = mh * P, mh * P + 2 * G * N
        moe = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": E, "top": top}, "shared": {"ff": sh}}
        rot = {"dims": 64, "base": 1e6, "scaling": {"factor": 8.0, "original": 8192, "fast": 32.0, "slow": 1.0}}
        raw_n = {"architecture": "Nipudra", "vocab": V, "width": H, "norm": {"eps": 1e-6}, "embedding": {"scale": H ** 0.5},
                 "logit_scale": 0.5, "logit_softcap": 40.0, "token_side": {"dim": side}, "layers": [
            {"type": "retention", "mixer": {"heads": rh, "dim": rd, "vdim": rd, "decay": [1.0 - 2.0 ** (-5 - 3 * i / rh) for i in range(rh)],
                                            "rot": {"dims": 64, "base": 1e6}}, "mlp": moe},
            {"type": "attention", "mixer": {"heads": nh, "kv_heads": nkv, "dim": hd, "vdim": hd, "scale": hd ** -0.5, "diff": 0.2, "conv": taps,
                                            "mask": {"size": win}, "rot": rot}, "mlp": moe},
            {"type": "mamba2", "mixer": {"heads": mh, "vdim": P, "state": N, "groups": G, "conv": taps, "norm_groups": G}, "mlp": moe}]}
        wh, wd, wr = H // 64, 64, 64
        trot = {"dims": 64, "base": 1e6, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}
        raw_t = {"architecture": "Tekarax", "vocab": V, "width": H, "norm": {"eps": 1e-6}, "layers": [
            {"type": "wkv", "mixer": {"heads": wh, "dim": wd, "decay_rank": wr}, "mlp": moe},
            {"type": "attention", "mixer": {"heads": 2 * nh, "kv_heads": 2 * nkv, "dim": hd, "vdim": hd, "scale": hd ** -0.5, "rot": trot}, "mlp": moe}]}
        raw_m = {"architecture": "Modovik", "vocab": V, "width": H, "norm": {"eps": 1e-6}, "layers": [
            {"type": "lightning", "mixer": {"heads": rh, "dim": rd, "vdim": rd, "decay": [1.0 - 2.0 ** (-5 - 3 * i / rh) for i in range(rh)]},
             "mlp": {"kind": "dense", "ff": 4 * H}}]}
        q_maps, k_maps = 2 * nh * hd, 2 * nkv * hd             # the attention's maps: each a head of the kernels

        def attention_pairs(Tn, B, before, window=None):
            first = np.arange(before, before + Tn // B)
            return B * float((np.minimum(first + 1, window) if window else first + 1).sum())

        def routed(Tn, n, gated):
            pairs, up = Tn * top, 2 if gated else 1
            used = min(E, pairs)
            w = {"experts_gate_up": {"bytes": n * (used * up * ff * H * 2 + pairs * (H + up * ff) * 2), "flops": 2.0 * n * up * pairs * H * ff},
                 "experts_down": {"bytes": n * (used * H * ff * 2 + pairs * (ff * 2 + H * 4)), "flops": 2.0 * n * pairs * H * ff},
                 "router": {"bytes": n * (E * H * 4 + Tn * H * 2 + pairs * H * (4 + 2) + Tn * H * 4), "flops": 2.0 * n * Tn * H * E}}
            if gated:
                w["gate_up"] = {"bytes": n * (2 * sh * H * 2 + Tn * (H + 2 * sh) * 2), "flops": 4.0 * n * Tn * H * sh}
            else:
                w["up"] = {"bytes": n * (sh * H * 2 + Tn * (H + sh) * 2), "flops": 2.0 * n * Tn * H * sh}
            w["down"] = {"bytes": n * (H * sh * 2 + Tn * (sh + H) * 2), "flops": 2.0 * n * Tn * H * sh}
            return w

        def tail(Tn, B):
            return {"head": {"bytes": V * H * 2 + B * (H * 2 + V * 4), "flops": 2.0 * B * H * V}, "embed": {"bytes": Tn * H * (2 + 4), "flops": 0}}

        def work_nipudra(Tn, B, before):
            proj = 4 * rh * rd + (q_maps + k_maps + k_maps) + (2 * inner + 2 * G * N + mh)      # q k v g | maps, values per map | z x B C dt
            cached = B * min(before + Tn // B, win + Tn // B)
            return {
                "qkv": {"bytes": proj * H * 2 + Tn * (3 * H + proj) * 2, "flops": 2.0 * Tn * H * proj},
                "short_conv": {"bytes": Tn * (q_maps + 2 * k_maps + conv_ch) * (2 + 2) + B * (taps - 1) * (q_maps + 2 * k_maps + conv_ch) * 8, "flops": 0},
                "linear_attention": {"bytes": Tn * 3 * rh * rd * 2 + Tn * rh * rd * 4 + B * 2 * rh * rd * rd * 4, "flops": 4.0 * Tn * rh * rd * rd},
                "recurrence": {"bytes": Tn * (conv_ch * 2 + inner * 4) + B * 2 * mh * N * P * 4, "flops": 6.0 * Tn * mh * N * P},
                "attention": {"bytes": cached * 2 * k_maps * 2 + 2 * Tn * q_maps * 2, "flops": 4.0 * 2 * nh * hd * attention_pairs(Tn, B, before, win)},
                "o": {"bytes": (rh * rd + nh * hd + inner) * H * 2 + Tn * (rh * rd + nh * hd + inner + 3 * H) * 2,
                      "flops": 2.0 * Tn * H * (rh * rd + nh * hd + inner)},
                "side": {"bytes": 3 * (2 * side * H * 2 + Tn * (2 * H + 3 * side) * 2), "flops": 3 * 4.0 * Tn * H * side},
                "activation": {"bytes": 3 * Tn * top * 2 * ff * 2 + 3 * Tn * 2 * sh * 2 + Tn * H * 2 * 2, "flops": 0},
                "norm": {"bytes": Tn * H * (2 + 2 + 4 + 4), "flops": 0, "per_launch": True},
                "gate": {"bytes": Tn * inner * (4 + 2 + 2) // 2, "flops": 0, "per_launch": True},
                "rotary+write": {"bytes": Tn * (q_maps + 2 * k_maps) * 2 * 2, "flops": 0, "per_launch": True},
                **routed(Tn, 3, False), **tail(Tn, B)}

        def work_tekarax(Tn, B, before):
            whd = wh * wd
            proj = 4 * whd + (q_maps + 2 * k_maps + 2 * nh)
            return {
                "qkv": {"bytes": proj * H * 2 + Tn * (5 * H + proj) * 2, "flops": 2.0 * Tn * H * proj},
                "decay": {"bytes": (wr * H + whd * wr) * 2 + Tn * (H + 2 * wr) * 2 + Tn * whd * 4, "flops": 2.0 * Tn * wr * (H + whd)},
                "recurrence": {"bytes": Tn * (H * 2 * 6 + whd * (2 * 5 + 4)) + B * (2 * wh * wd * wd + 2 * H) * 4, "flops": 6.0 * Tn * wh * wd * wd},
                "attention": {"bytes": B * (before + Tn // B) * 2 * k_maps * 2 + 2 * Tn * q_maps * 2, "flops": 4.0 * 2 * nh * hd * attention_pairs(Tn, B, before)},
                "o": {"bytes": (whd + q_maps) * H * 2 + Tn * (whd + q_maps + 2 * H) * 2, "flops": 2.0 * Tn * H * (whd + q_maps)},
                "residual_gate": {"bytes": 4 * (H * H * 2 + Tn * 2 * H * 2), "flops": 2.0 * 4 * Tn * H * H},
                "activation": {"bytes": 2 * Tn * top * 3 * ff * 2 + 2 * Tn * 3 * sh * 2 + Tn * wr * 4, "flops": 0},
                "norm": {"bytes": Tn * H * (2 + 2 + 4 + 4), "flops": 0, "per_launch": True},
                "gate": {"bytes": Tn * q_maps * (2 + 2), "flops": 0, "per_launch": True},
                "rotary+write": {"bytes": Tn * (q_maps + 2 * k_maps) * 2 * 2, "flops": 0, "per_launch": True},
                **routed(Tn, 2, True), **tail(Tn, B)}

        def work_modovik(Tn, B, before):
            I = 4 * H
            return {
                "qkv": {"bytes": 4 * rh * rd * H * 2 + Tn * (H + 4 * rh * rd) * 2, "flops": 2.0 * Tn * H * 4 * rh * rd},
                "linear_attention": {"bytes": Tn * 3 * rh * rd * 2 + Tn * rh * rd * 4 + B * 2 * rh * rd * rd * 4, "flops": 4.0 * Tn * rh * rd * rd},
                "o": {"bytes": rh * rd * H * 2 + Tn * (rh * rd + H) * 2, "flops": 2.0 * Tn * H * rh * rd},
                "up": {"bytes": I * H * 2 + Tn * (H + I) * 2, "flops": 2.0 * Tn * H * I},
                "down": {"bytes": H * I * 2 + Tn * (I + H) * 2, "flops": 2.0 * Tn * H * I},
                "activation": {"bytes": Tn * I * 4, "flops": 0},
                "norm": {"bytes": Tn * H * (2 + 4 + 4 + 2), "flops": 0, "per_launch": True},
                "gate": {"bytes": Tn * rh * rd * (4 + 2 + 2), "flops": 0, "per_launch": True},
                **tail(Tn, B)}

        block = {"sizes": dict(z, retention_heads=rh, state_space_heads=mh, state=N, groups=G), "models": {}}
        for name, raw, work in (("nipudra", raw_n, work_nipudra), ("tekarax", raw_t, work_tekarax), ("modovik", raw_m, work_modovik)):
            block["models"][name] = dict(layers=len(raw["layers"]), **_measure_design(config_from_dict(raw), work, args, peaks, V, T, ctx_len, rng))
        out["sizes"][tag] = block
    return out


def run_gadopel(args) -> dict:
    """``--workload gadopel``: the Gadopel design (random weights) at two sets of layer sizes, two layers that run twice
    (latent attention with a sink and a gate per head; grouped-query attention over a window beside kept first tokens;
    each beside a relu-gated feed-forward; the stream fed with the embedding again before each pass), beside the
    package's closest layers at equal sizes, run as often: Pivinex's latent attention beside a gelu-gated feed-forward,
    and Tekarax's grouped-query attention with a dense feed-forward.  A 2,048-token prompt step and decode steps at
    batch 8 and 64 with 2,048 tokens of context, device-timed, and per kernel class the device time of one such step with
    the fraction of the measured peak."""
    import numpy as np

    from pyre_b200.config import config_from_dict

    peaks = load_peaks()
    V = 32768
    sizes = {
        # width; heads of 128 + 64, values of 128, latent; key/value heads of the grouped-query layer; window, kept
        # first tokens; feed-forward
        "2k": dict(H=2048, nh=16, dn=128, dr=64, dv=128, kr=256, nkv=4, win=1024, keep=64, I=8192),
        "3.5k": dict(H=3584, nh=28, dn=128, dr=64, dv=128, kr=512, nkv=4, win=4096, keep=128, I=18944),
    }
    T, ctx_len, times = PROMPT_LEN, 2048, 2
    rng = np.random.default_rng(0)
    out = {"workload": "gadopel", "peaks": peaks, "prompt": T, "decode_context": ctx_len, "sizes": {}}
    for tag, z in sizes.items():
        H, nh, dn, dr, dv, kr, nkv, win, keep, I = (z[k] for k in ("H", "nh", "dn", "dr", "dv", "kr", "nkv", "win", "keep", "I"))
        row, qr = kr + dr, 768
        scaling = {"factor": 8.0, "original": 8192, "fast": 32.0, "slow": 1.0}
        raw_g = {"architecture": "Gadopel", "vocab": V, "width": H, "norm": {"eps": 1e-6}, "loop": {"start": 0, "stop": 2, "times": times}, "layers": [
            {"type": "latent_attention", "mixer": {"heads": nh, "dim": dn, "rot_dim": dr, "vdim": dv, "kv_rank": kr, "scale": (dn + dr) ** -0.5,
                                                   "rot": {"dims": dr, "base": 1e6}}, "mlp": {"kind": "dense", "ff": I}},
            {"type": "attention", "mixer": {"heads": nh, "kv_heads": nkv, "dim": dn, "vdim": dv, "scale": dn ** -0.5, "mask": {"size": win, "keep_first": keep},
                                            "rot": {"dims": dn, "base": 1e6, "scaling": scaling}}, "mlp": {"kind": "dense", "ff": I}}]}
        raw_p = {"architecture": "Pivinex", "vocab": V, "width": H, "norm": {"eps": 1e-6}, "residual_mult": 0.5,
                 "loop": {"start": 0, "stop": 1, "times": times}, "layers": [
            {"type": "latent_attention", "mixer": {"heads": nh, "dim": dn, "rot_dim": dr, "vdim": dv, "q_rank": qr, "kv_rank": kr, "scale": (dn + dr) ** -0.5,
                                                   "mask": {"size": 1 << 20}, "rot": {"dims": dr, "base": 1e6}}, "mlp": {"kind": "dense", "ff": I}}]}
        raw_t = {"architecture": "Tekarax", "vocab": V, "width": H, "norm": {"eps": 1e-6}, "loop": {"start": 0, "stop": 1, "times": times}, "layers": [
            {"type": "attention", "mixer": {"heads": nh, "kv_heads": nkv, "dim": dn, "vdim": dv, "scale": dn ** -0.5,
                                            "rot": {"dims": dn, "base": 1e6, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}},
             "mlp": {"kind": "dense", "ff": I}}]}
        q, kv = nh * dn, nkv * dn

        def pairs(Tn, B, before, window=None, kept=0):
            """query-key pairs of a step of B entries, ``before`` tokens cached each"""
            seen = np.arange(before, before + Tn // B) + 1
            return B * float((np.minimum(seen, window + kept) if window else seen).sum())

        def latent(Tn, B, before, n):
            cached = B * (before + Tn // B)
            return {
                "absorb": {"bytes": n * (nh * dn * kr * 2 + Tn * nh * (dn + kr) * 2), "flops": 2.0 * n * Tn * nh * dn * kr},
                "latent_attention": {"bytes": n * (cached * row * 2 + Tn * nh * (row + kr) * 2), "flops": 2.0 * n * nh * (kr + dr + kr) * pairs(Tn, B, before)},
                "v_up": {"bytes": n * (nh * dv * kr * 2 + Tn * nh * (kr + dv) * 2), "flops": 2.0 * n * Tn * nh * kr * dv}}

        def product(rows, cols, Tn, n):
            return {"bytes": n * (rows * cols * 2 + Tn * (rows + cols) * 2), "flops": 2.0 * n * Tn * rows * cols}

        def tail(Tn, B):
            return {"head": {"bytes": V * H * 2 + B * (H * 2 + V * 4), "flops": 2.0 * B * H * V}, "embed": {"bytes": Tn * H * (2 + 4), "flops": 0}}

        def gated(Tn, n):
            return {"gate_up": {"bytes": n * (2 * I * H * 2 + Tn * (H + I) * 2), "flops": 4.0 * n * Tn * H * I}, "down": product(I, H, Tn, n)}

        def work_gadopel(Tn, B, before):
            cols = nh * (dn + dr) + kr + dr + nh + (q + 2 * kv)
            per = Tn // B
            seen = B * min(before + per, win + keep + per)
            return {
                "qkv": {"bytes": times * (cols * H * 2 + Tn * (2 * H + cols) * 2), "flops": 2.0 * times * Tn * H * cols},
                "attention": {"bytes": times * (seen * 2 * kv * 2 + 2 * Tn * q * 2), "flops": 4.0 * times * nh * dn * pairs(Tn, B, before, win, keep)},
                "o": product(nh * dv, H, Tn, 2 * times),
                # the embedding's half once per step, the stream's half once per pass; fp32 results
                "feed_again": {"bytes": (times + 1) * (H * H * 2 + Tn * H * (2 + 4)), "flops": 2.0 * (times + 1) * Tn * H * H},
                "norm": {"bytes": Tn * H * (2 + 2 + 4 + 4 + 2 + 2), "flops": 0, "per_launch": True},
                # rotated parts of the queries, latent rows; whole heads of the grouped-query layer: read and written once
                "rotary+write": {"bytes": times * Tn * (nh * dr + row + q + 2 * kv) * 4, "flops": 0},
                **latent(Tn, B, before, times), **gated(Tn, 2 * times), **tail(Tn, B)}

        def work_pivinex(Tn, B, before):
            cols = qr + kr + dr
            return {
                "qkv": product(cols, H, Tn, times), "q_up": product(nh * (dn + dr), qr, Tn, times), "o": product(nh * dv, H, Tn, times),
                "norm": {"bytes": Tn * H * (2 + 2 + 4 + 4 + 2), "flops": 0, "per_launch": True},
                "rotary+write": {"bytes": times * Tn * (cols + qr + row + 2 * nh * dr) * 2, "flops": 0},
                **latent(Tn, B, before, times), **gated(Tn, times), **tail(Tn, B)}

        def work_tekarax(Tn, B, before):
            cols = q + 2 * kv + nh
            return {
                "qkv": product(cols, H, Tn, times), "o": product(q, H, Tn, times), "up": product(I, H, Tn, times), "down": product(I, H, Tn, times),
                "attention": {"bytes": times * (B * (before + Tn // B) * 2 * kv * 2 + 2 * Tn * q * 2), "flops": 4.0 * times * nh * dn * pairs(Tn, B, before)},
                "residual_gate": product(H, H, Tn, 2 * times),
                "activation": {"bytes": times * Tn * I * 4, "flops": 0},
                "norm": {"bytes": Tn * H * (2 + 2 + 4 + 4), "flops": 0, "per_launch": True},
                "gate": {"bytes": Tn * q * (2 + 2), "flops": 0, "per_launch": True},
                "rotary+write": {"bytes": times * Tn * (q + 2 * kv) * 2 * 2, "flops": 0},
                **tail(Tn, B)}

        block = {"sizes": dict(z), "models": {}}
        for name, raw, work in (("gadopel", raw_g, work_gadopel), ("pivinex", raw_p, work_pivinex), ("tekarax", raw_t, work_tekarax)):
            block["models"][name] = dict(layers=len(raw["layers"]), times=times, **_measure_design(config_from_dict(raw), work, args, peaks, V, T, ctx_len, rng))
        out["sizes"][tag] = block
    return out


def run_gugidra(args) -> dict:
    """``--workload gugidra``: the Gugidra design (random weights) at two sets of layer sizes, two layers that run twice
    (gated linear attention with a clamped dense feed-forward; attention over its own keys beside a matrix memory, with
    experts chosen in groups and a shared one), beside the package's closest layers at equal sizes: Tekarax's recurrent
    layer with a dense feed-forward and its attention layer with routed experts, run as often, and two of Modovik's
    constant-decay layers with dense feed-forwards, whose state is the matrix memory's.  A 2,048-token prompt step and
    decode steps at batch 8 and 64 with 2,048 tokens of context, device-timed, and per kernel class the device time of one
    such step with the fraction of the measured peak."""
    import numpy as np

    from pyre_b200.config import config_from_dict

    peaks = load_peaks()
    V = 32768
    sizes = {
        # width; attention heads of 128 over key/value heads (and as many memory heads of 128 x 128); recurrent head size and
        # the decay map's inner size; dense feed-forward; experts in groups of which some are kept, chosen, their size, shared
        "2k": dict(H=2048, nh=16, nkv=4, hd=128, wd=64, wr=64, I=8192, E=32, groups=8, keep=4, top=4, ff=1024, sh=2048),
        "3.5k": dict(H=3584, nh=28, nkv=4, hd=128, wd=64, wr=96, I=18944, E=64, groups=8, keep=4, top=6, ff=1408, sh=2816),
    }
    T, ctx_len, times = PROMPT_LEN, 2048, 2
    rng = np.random.default_rng(0)
    out = {"workload": "gugidra", "peaks": peaks, "prompt": T, "decode_context": ctx_len, "sizes": {}}
    for tag, z in sizes.items():
        H, nh, nkv, hd, wd, wr, I, E, top, ff, sh = (z[k] for k in ("H", "nh", "nkv", "hd", "wd", "wr", "I", "E", "top", "ff", "sh"))
        wh = H // wd
        q, kv, whd = nh * hd, nkv * hd, wh * wd
        dense = {"kind": "dense", "ff": I}
        loop = {"start": 0, "stop": 2, "times": times}
        raw_g = {"architecture": "Gugidra", "vocab": V, "width": H, "norm": {"eps": 1e-6}, "embedding": {"scale": H ** 0.5},
                 "logit_softcap": 30.0, "loop": loop, "layers": [
            {"type": "gla", "mixer": {"heads": wh, "dim": wd, "vdim": wd, "tau": 16.0, "decay_rank": wr}, "mlp": dict(dense, limit=7.0)},
            {"type": "parallel", "mixer": {
                "left": {"heads": nh, "kv_heads": nkv, "dim": hd, "vdim": hd, "scale": hd ** -0.5, "rot": {"dims": hd, "base": 1e6}},
                "right": {"heads": nh, "dim": hd, "vdim": hd, "gate_cap": 15.0}, "left_scale": 0.7, "right_scale": 0.8},
             "mlp": {"kind": "moe", "expert": {"ff": ff, "limit": 7.0}, "router": {"experts": E, "top": top, "groups": {"count": z["groups"], "keep": z["keep"]}},
                     "shared": {"ff": sh, "limit": 7.0}}}]}
        raw_t = {"architecture": "Tekarax", "vocab": V, "width": H, "norm": {"eps": 1e-6}, "loop": loop, "layers": [
            {"type": "wkv", "mixer": {"heads": wh, "dim": wd, "decay_rank": wr}, "mlp": dense},
            {"type": "attention", "mixer": {"heads": nh, "kv_heads": nkv, "dim": hd, "vdim": hd, "scale": hd ** -0.5, "rot": {"dims": hd, "base": 1e6}},
             "mlp": {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": E, "top": top}, "shared": {"ff": sh}}}]}
        raw_m = {"architecture": "Modovik", "vocab": V, "width": H, "norm": {"eps": 1e-6}, "layers": [
            {"type": "lightning", "mixer": {"heads": nh, "dim": hd, "vdim": hd, "decay": [1.0 - 2.0 ** (-5 - 3 * i / nh) for i in range(nh)]},
             "mlp": dense}] * times}

        def pairs(Tn, B, before):
            return B * float((np.arange(before, before + Tn // B) + 1).sum())

        def product(rows, cols, Tn, n):
            return {"bytes": n * (rows * cols * 2 + Tn * (rows + cols) * 2), "flops": 2.0 * n * Tn * rows * cols}

        def state(Tn, B, heads, dim, n, extra=0):
            """a recurrence over [dim, dim] states: q, k, v in, fp32 values out (and ``extra`` bytes per token), the state in and out"""
            w = heads * dim
            return {"bytes": n * (Tn * (w * (3 * 2 + 4) + extra) + B * 2 * heads * dim * dim * 4), "flops": 4.0 * n * Tn * heads * dim * dim}

        def attention(Tn, B, before, n):
            return {"bytes": n * (B * (before + Tn // B) * 2 * kv * 2 + 2 * Tn * q * 2), "flops": 4.0 * n * nh * hd * pairs(Tn, B, before)}

        def routed(Tn, n):
            chosen = Tn * top
            used = min(E, chosen)
            return {"experts_gate_up": {"bytes": n * (used * 2 * ff * H * 2 + chosen * (H + 2 * ff) * 2), "flops": 4.0 * n * chosen * H * ff},
                    "experts_down": {"bytes": n * (used * H * ff * 2 + chosen * (ff * 2 + H * 4)), "flops": 2.0 * n * chosen * H * ff},
                    "router": {"bytes": n * (E * H * 4 + Tn * H * 2 + chosen * H * 4 + Tn * H * 4), "flops": 2.0 * n * Tn * H * E}}

        def tail(Tn, B):
            return {"head": {"bytes": V * H * 2 + B * (H * 2 + V * 4), "flops": 2.0 * B * H * V}, "embed": {"bytes": Tn * H * (2 + 4), "flops": 0}}

        def work_gugidra(Tn, B, before):
            cols = 4 * whd + wr + q + kv + 4 * q
            return {
                "qkv": {"bytes": times * (cols * H * 2 + Tn * (2 * H + cols) * 2), "flops": 2.0 * times * Tn * H * cols},
                "gates": {"bytes": times * (2 * nh * H * 2 + Tn * (H * 2 + 2 * nh * 4)), "flops": 2.0 * times * Tn * H * 2 * nh},
                "decay": {"bytes": times * (whd * wr * 4 + Tn * (wr * 2 + whd * 4)), "flops": 2.0 * times * Tn * wr * whd},
                "recurrence": state(Tn, B, wh, wd, times, extra=whd * 4), "matrix_memory": state(Tn, B, nh, hd, times, extra=nh * 12),
                "attention": attention(Tn, B, before, times),
                "o": {"bytes": times * ((whd + 2 * q) * H * 2 + Tn * (whd + 2 * q + 2 * H) * 2), "flops": 2.0 * times * Tn * H * (whd + 2 * q)},
                "gate_up": {"bytes": times * (2 * (I + sh) * H * 2 + Tn * (2 * H + I + sh) * 2), "flops": 4.0 * times * Tn * H * (I + sh)},
                "down": {"bytes": times * ((I + sh) * H * 2 + Tn * (I + sh + 2 * H) * 2), "flops": 2.0 * times * Tn * H * (I + sh)},
                "activation": {"bytes": times * Tn * top * 3 * ff * 2, "flops": 0},
                "norm": {"bytes": Tn * H * (2 + 4 + 4 + 2), "flops": 0, "per_launch": True},
                "gate": {"bytes": times * Tn * ((whd + q) * (4 + 2 + 2) + q * (2 + 2)), "flops": 0},
                "rotary+write": {"bytes": times * Tn * (q + 2 * kv) * 2 * 2, "flops": 0},
                **routed(Tn, times), **tail(Tn, B)}

        def work_tekarax(Tn, B, before):
            cols = 4 * whd + q + 2 * kv + nh
            return {
                "qkv": {"bytes": times * (cols * H * 2 + Tn * (5 * H + cols) * 2), "flops": 2.0 * times * Tn * H * cols},
                "decay": {"bytes": times * ((wr * H + whd * wr) * 2 + Tn * (H + 2 * wr) * 2 + Tn * whd * 4), "flops": 2.0 * times * Tn * wr * (H + whd)},
                "recurrence": {"bytes": times * (Tn * (H * 2 * 6 + whd * (2 * 5 + 4)) + B * (2 * wh * wd * wd + 2 * H) * 4), "flops": 6.0 * times * Tn * wh * wd * wd},
                "attention": attention(Tn, B, before, times),
                "o": {"bytes": times * ((whd + q) * H * 2 + Tn * (whd + q + 2 * H) * 2), "flops": 2.0 * times * Tn * H * (whd + q)},
                "up": product(I, H, Tn, times), "gate_up": product(2 * sh, H, Tn, times),
                "down": {"bytes": times * ((I + sh) * H * 2 + Tn * (I + sh + 2 * H) * 2), "flops": 2.0 * times * Tn * H * (I + sh)},
                "residual_gate": product(H, H, Tn, 4 * times),
                # the experts' activation; the dense feed-forward's runs in the class of its product
                "activation": {"bytes": times * Tn * top * 3 * ff * 2, "flops": 0},
                "norm": {"bytes": Tn * H * (2 + 2 + 4 + 4), "flops": 0, "per_launch": True},
                "gate": {"bytes": Tn * q * (2 + 2), "flops": 0, "per_launch": True},
                "rotary+write": {"bytes": times * Tn * (q + 2 * kv) * 2 * 2, "flops": 0},
                **routed(Tn, times), **tail(Tn, B)}

        def work_modovik(Tn, B, before):
            return {
                "qkv": product(4 * q, H, Tn, times), "linear_attention": state(Tn, B, nh, hd, times), "o": product(q, H, Tn, times),
                "up": product(I, H, Tn, times), "down": product(I, H, Tn, times), "activation": {"bytes": times * Tn * I * 4, "flops": 0},
                "norm": {"bytes": Tn * H * (2 + 4 + 4 + 2), "flops": 0, "per_launch": True},
                "gate": {"bytes": Tn * q * (4 + 2 + 2), "flops": 0, "per_launch": True}, **tail(Tn, B)}

        block = {"sizes": dict(z, recurrent_heads=wh), "models": {}}
        for name, raw, work in (("gugidra", raw_g, work_gugidra), ("tekarax", raw_t, work_tekarax), ("modovik", raw_m, work_modovik)):
            block["models"][name] = dict(layers=len(raw["layers"]), times=1 if name == "modovik" else times,
                                         **_measure_design(config_from_dict(raw), work, args, peaks, V, T, ctx_len, rng))
        out["sizes"][tag] = block
    return out


def run_sweep(args) -> dict:
    """Decode throughput over a grid of batch sizes and context lengths and prefill throughput over
    several portion lengths on the 7B shape, each with its fraction of the roofline (device-timed,
    the same way as the headline numbers).  One JSON object; not part of the one-line contract."""
    import numpy as np
    import torch

    from pyre_b200 import Engine
    from pyre_b200.config import config_from_dict
    from pyre_b200.engine.step import StepEntry
    from pyre_b200.kernels import ops

    peaks = load_peaks()
    cfg_raw = dict(CONFIG_7B)
    layers = args.layers or cfg_raw["num_hidden_layers"]
    cfg_raw["num_hidden_layers"] = layers
    cfg_raw["max_position_embeddings"] = 40960
    cfg = config_from_dict(cfg_raw)
    weight_bytes, kv_per_token, flops = model_numbers(cfg_raw, layers)
    grid = [(1, 512), (1, 8192), (1, 32768), (8, 512), (8, 2048), (8, 8192), (8, 32768), (32, 2048), (64, 512), (64, 2048),
            (64, 8192), (128, 2048)]
    biggest = max(b * (c + SETTLE_STEPS + 64) for b, c in grid)
    eng = Engine(config=cfg, seed=0, dtype="bfloat16", page_size=PAGE_SIZE, max_cache_tokens=biggest + 8192,
                 max_num_seqs=128, max_num_batched_tokens=8192, prefill_chunk=8192, max_model_len=40960)
    st, cache = eng.stepper, eng.cache
    rng = np.random.default_rng(0)
    vocab = cfg.vocab_size

    def ev():
        return torch.cuda.Event(enable_timing=True)

    decode = []
    for batch, ctx in grid:
        reqs = [("d", batch, ctx, i) for i in range(batch)]
        for r in reqs:
            cache.begin(r)
            for lo in range(0, ctx, 8192):
                st.step([StepEntry(r, rng.integers(0, vocab, min(8192, ctx - lo)).tolist(), [])])
        n_warm, n_steps = SETTLE_STEPS + 8, 32
        toks = rng.integers(0, vocab, (n_warm + n_steps, batch))
        for k in range(n_warm):
            ops.sample(st.step([StepEntry(r, [int(toks[k, i])], [0]) for i, r in enumerate(reqs)]))
        torch.cuda.synchronize()
        a, b = ev(), ev()
        a.record()
        for k in range(n_warm, n_warm + n_steps):
            ops.sample(st.step([StepEntry(r, [int(toks[k, i])], [0]) for i, r in enumerate(reqs)]))
        b.record()
        torch.cuda.synchronize()
        ms = a.elapsed_time(b) / n_steps
        step_bytes = weight_bytes + kv_per_token * (ctx + n_warm + n_steps / 2) * batch
        decode.append({"batch": batch, "context": ctx, "ms_per_step": round(ms, 3), "tok_s": round(batch / ms * 1e3, 1),
                       "hbm_frac": round(step_bytes / (ms * 1e-3) / 1e9 / peaks["hbm_gbs"], 3)})
        for r in reqs:
            cache.end(r)
    prefill = []
    for T, start in ((512, 0), (2048, 0), (4096, 0), (8192, 0), (2048, 8192), (2048, 30720), (512, 30720), (128, 30720)):
        times = []
        for rep in range(4):
            r = ("p", T, start, rep)
            cache.begin(r)
            for lo in range(0, start, 8192):
                st.step([StepEntry(r, rng.integers(0, vocab, min(8192, start - lo)).tolist(), [])])
            ids = rng.integers(0, vocab, T).tolist()
            torch.cuda.synchronize()
            a, b = ev(), ev()
            a.record()
            ops.sample(st.step([StepEntry(r, ids, [T - 1])]))
            b.record()
            torch.cuda.synchronize()
            times.append(a.elapsed_time(b))
            cache.end(r)
        ms = sorted(times[1:])[len(times[1:]) // 2]
        prefill.append({"tokens": T, "context_before": start, "ms": round(ms, 3), "tok_s": round(T / ms * 1e3, 1),
                        "flops_frac": round(flops(T, start, 1) / (ms * 1e-3) / (peaks["bf16_tflops"] * 1e12), 3)})
    cache.check()
    st.check_device_errors()
    return {"workload": "sweep", "layers": layers, "peaks": peaks, "decode": decode, "prefill": prefill}


def environment() -> dict:
    """Where a number was measured, recorded with it as the reference's harness does (bench/harness.py:49-67):
    GPU, compute capability, torch and CUDA versions, the checkout's commit, the time."""
    env = {"gpu": None, "capability": None, "torch": None, "cuda": None, "git": None,
           "time": time.strftime("%Y-%m-%dT%H:%M:%SZ", time.gmtime())}
    try:
        import torch
        env["torch"], env["cuda"] = torch.__version__, torch.version.cuda
        if torch.cuda.is_available():
            env["gpu"] = torch.cuda.get_device_name(0)
            env["capability"] = ".".join(str(v) for v in torch.cuda.get_device_capability(0))
    except Exception:       # the record must never cost the measurement
        pass
    try:
        out = subprocess.run(["git", "-C", str(ROOT), "rev-parse", "--short", "HEAD"], capture_output=True, text=True,
                             timeout=10)
        env["git"] = out.stdout.strip() or None
    except (OSError, subprocess.SubprocessError):
        pass
    return env


def run_reference(args) -> dict:
    from baseline import reference_arm
    layers = args.layers or CONFIG_7B["num_hidden_layers"]
    return reference_arm.run(args, CONFIG_7B, PROMPT_LEN,
                             bench_config(CONFIG_7B, layers, CONFIG_7B["num_hidden_layers"], args.batch))


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=4)
    ap.add_argument("--impl", choices=["ours", "reference"], default="ours")
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--layers", type=int, default=0, help="fewer layers than the configuration has (0 = all)")
    ap.add_argument("--prefill-reps", type=int, default=5)
    ap.add_argument("--skip-points", action="store_true", help="leave out decode at batch 1 and 64")
    ap.add_argument("--skip-sizes", action="store_true",
                    help="leave out the points at longer contexts and at the 14B and 32B shapes")
    ap.add_argument("--no-per-kernel", action="store_true",
                    help="leave out the `kernels` block (device time, bytes or flops and fraction of the peak per kernel class)")
    ap.add_argument("--workload", choices=["serve14b", "mixed32b", "sweep", "modovik", "pivinex", "tekarax", "nipudra", "gadopel", "gugidra"], default=None,
                    help="run one of the two other baseline workloads, a sweep over batch sizes, context lengths and "
                         "portion lengths on the 7B shape, the Modovik or the Pivinex design beside the Qwen2.5 decoder at "
                         "equal layer sizes, the Tekarax design beside the closest layers of those two, the Nipudra design beside the closest "
                         "layers of Tekarax and Modovik, the Gadopel design beside the closest layers of Pivinex and Tekarax, or the Gugidra design beside the closest layers of Tekarax and Modovik, instead (prints its own JSON line)")
    ap.add_argument("--cache-fraction", type=float, default=1.0,
                    help="serve14b: cache capacity as a fraction of what all requests need at once (< 1 forces preemption)")
    args = ap.parse_args()
    if args.gpus != 1:
        print(f"bench.py measures a single-GPU engine: --gpus {args.gpus} is not supported, run with --gpus 1")
        return 2
    if args.workload:
        result = run_sweep(args) if args.workload == "sweep" else run_modovik(args) if args.workload == "modovik" else \
            run_pivinex(args) if args.workload == "pivinex" else run_tekarax(args) if args.workload == "tekarax" else run_nipudra(args) if args.workload == "nipudra" else \
            run_gadopel(args) if args.workload == "gadopel" else run_gugidra(args) if args.workload == "gugidra" else run_workload(args)
        result["env"] = environment()
        print(json.dumps(result))
        return 0
    result = run_reference(args) if args.impl == "reference" else run_ours(args)
    if "unavailable" not in result:
        result["env"] = environment()
    print(json.dumps(result))
    return 0


if __name__ == "__main__":
    sys.exit(main())
