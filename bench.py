#!/usr/bin/env python3
"""Decode and prefill throughput of the engine at Qwen3-8B layer sizes, random
bf16 weights, one GPU.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl reference]

One JSON line on stdout.  ``value`` is decoded tokens per second at batch 8
(device-timed, sampled tokens fed back on the device), timed at contexts of 2,048,
3,072 and 4,095 tokens and averaged: the run from 2,048-token prompts to the 4,096
context; ``e2e`` is decode through ``Engine.generate`` with host tokens in and out
every step; ``prefill`` is one 2,048-token prompt; ``roofline`` relates the decode
step's mandatory HBM reads to the measured copy bandwidth; ``points`` holds, as flat
numbers, each context of the headline, decode at batch 1 and 64, and the baseline's
other configurations (Qwen3-0.6B sizes incl. the 64 unequal prompts through
``generate``, Qwen3-32B sizes with a cache for 64 x 4,096 tokens); ``kernels`` gives
every operation of a prefill and of a decode step by CUDA events with its fraction of
the measured peak; ``cpu_baseline`` times the plain implementation on the two tiny
configurations.
"""
from __future__ import annotations

import argparse
import gc
import json
import os
import statistics
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

QWEN3_8B = {
    "architectures": ["Qwen3ForCausalLM"], "num_hidden_layers": 36, "hidden_size": 4096,
    "num_attention_heads": 32, "num_key_value_heads": 8, "head_dim": 128, "intermediate_size": 12288,
    "vocab_size": 151936, "rope_theta": 1000000.0, "rms_norm_eps": 1e-6, "tie_word_embeddings": False,
    "max_position_embeddings": 40960, "hidden_act": "silu",
}
# the other layer sizes that the baseline's configurations name (--sizes); the default run stays Qwen3-8B
OTHER_SIZES = {
    "0.6b": dict(QWEN3_8B, num_hidden_layers=28, hidden_size=1024, num_attention_heads=16, num_key_value_heads=8,
                 intermediate_size=3072, tie_word_embeddings=True),
    "32b": dict(QWEN3_8B, num_hidden_layers=64, hidden_size=5120, num_attention_heads=64, num_key_value_heads=8,
                intermediate_size=25600),
}
PROMPT_LEN = 2048
CONTEXT = 4096
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


def peaks() -> dict:
    p = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.isfile(p):
        try:
            with open(p) as f:
                d = json.load(f)
            out = dict(FALLBACK_PEAKS)
            for k in ("hbm_gbs", "bf16_tflops", "bf16_tflops_sustained"):
                if isinstance(d.get(k), (int, float)):
                    out[k] = float(d[k])
            out["source"] = "measured"
            return out
        except (OSError, ValueError):
            pass
    return dict(FALLBACK_PEAKS)


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while a region runs."""
    Q = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
         "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.rows = []
        self.proc = None

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", "0", f"--query-gpu={self.Q}",
                                          "--format=csv,noheader,nounits", "-lms", "100"],
                                         stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            self.t = threading.Thread(target=self._read, daemon=True)
            self.t.start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            parts = [p.strip() for p in line.split(",")]
            if len(parts) == 6:
                self.rows.append(parts)

    def stop(self) -> dict:
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        self.proc.terminate()
        try:
            self.proc.wait(timeout=5)
        except subprocess.TimeoutExpired:
            self.proc.kill()
        sm, mx, reasons = [], None, set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for r in self.rows:
            try:
                sm.append(float(r[0]))
                mx = float(r[1])
            except ValueError:
                continue
            for n, v in zip(names, r[2:]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        return {"sm_mhz": statistics.median(sm) if sm else None, "sm_max_mhz": mx, "reasons": sorted(reasons),
                "samples": len(sm)}


def model_numbers(cfg, layers: int):
    """Bytes of weights a decode step reads once and FLOPs per token of the linears."""
    H, I, V = cfg.hidden_size, cfg.intermediate_size, cfg.vocab_size
    Q, KV = cfg.num_attention_heads * cfg.head_dim, cfg.num_key_value_heads * cfg.head_dim
    per_layer = (Q + 2 * KV) * H + H * Q + 2 * I * H + H * I
    norms = layers * (2 * H + 2 * cfg.head_dim) + H
    weight_bytes = 2 * (layers * per_layer + V * H) + 4 * norms
    kv_bytes_per_token = layers * 2 * KV * 2
    return per_layer, weight_bytes, kv_bytes_per_token


CONTEXTS = (2048, 3072, 4095)      # where decode is timed: the start, the middle and the end of the run


class Runner:
    """One set of layer sizes: builds engines as the cases need them and times decode
    (device-timed, tokens fed back on the device), the same through ``Engine.generate``,
    prefill, and every operation of a step by CUDA events."""

    def __init__(self, sizes: str, layers, args, pk):
        import torch
        from zlm_b200.registry import config_from_dict
        from zlm_b200.sampling import SamplingParams
        self.torch = torch
        self.args, self.pk, self.sizes = args, pk, sizes
        d = dict(OTHER_SIZES.get(sizes, QWEN3_8B))
        self.full_layers = d["num_hidden_layers"]
        self.layers = self.full_layers if layers is None else layers
        d["num_hidden_layers"] = self.layers
        self.cfg = config_from_dict(d)
        self.per_layer, self.weight_bytes, self.kv_per_tok = model_numbers(self.cfg, self.layers)
        self.greedy = SamplingParams()
        self.g = torch.Generator().manual_seed(0)
        self.eng = None
        self.shape = None

    # ---- engines ------------------------------------------------------------------
    def engine(self, batch: int, tokens_per_seq: int):
        """An engine whose cache holds ``batch`` sequences of ``tokens_per_seq`` tokens (kept
        while it is large enough)."""
        torch = self.torch
        from zlm_b200 import Engine
        need = (batch, batch * tokens_per_seq)
        if self.eng is not None and self.shape[0] >= need[0] and self.shape[1] >= need[1]:
            return self.eng
        self.drop()
        e = Engine.from_random(self.cfg, seed=0, dtype="bfloat16", device="cuda:0", max_tokens=need[1],
                               max_batch=batch, max_seq_len=CONTEXT,
                               max_step_tokens=max(8 * CONTEXT, batch * PROMPT_LEN))      # `generate` takes all prompts in one step
        if self.args.pdl or self.args.no_pdl:
            e.decoder.use_pdl = bool(self.args.pdl)
        self.eng, self.shape = e, need
        return e

    def drop(self):
        if self.eng is not None:
            self.eng = None
            gc.collect()
            self.torch.cuda.empty_cache()

    def prompts(self, n: int, length: int):
        return [self.torch.randint(0, self.cfg.vocab_size, (length,), generator=self.g).tolist() for _ in range(n)]

    def prefill(self, eng, ps, chunk_tokens=8 * 2048):
        """Prompts into fresh slots, a few at a time; returns (slots, first sampled tokens)."""
        slots = [eng.new_sequence() for _ in ps]
        per = max(1, chunk_tokens // max(len(p) for p in ps))
        first = []
        for i in range(0, len(ps), per):
            first += eng.prefill_sample(slots[i:i + per], ps[i:i + per], self.greedy,
                                        list(range(i, i + len(ps[i:i + per]))))
        return slots, first

    # ---- decode ---------------------------------------------------------------------
    def decode_at(self, batch: int, context: int, steps: int, warmup: int, clocks=None) -> dict:
        """``steps`` decode steps of ``batch`` sequences that hold about ``context`` tokens,
        timed on the device around the whole run of steps."""
        torch = self.torch
        start = max(1, min(context, CONTEXT - warmup - steps))    # the timed steps end inside the context
        eng = self.engine(batch, CONTEXT)
        slots, first = self.prefill(eng, self.prompts(batch, start))
        dec, k = eng.decoder, eng.rt.k
        dec.step(slots, first, self.greedy)
        for _ in range(max(0, warmup - 1)):
            dec.step(slots, None, self.greedy)
        torch.cuda.synchronize()
        if clocks:
            clocks.start()
        ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        ctx0 = eng.length(slots[0])
        ev0.record()
        for _ in range(steps):
            dec.step(slots, None, self.greedy)
        ev1.record()
        torch.cuda.synchronize()
        ms = ev0.elapsed_time(ev1) / steps
        for sl in slots:
            eng.release(sl)
        eng.check(sync=True)
        mean_ctx = ctx0 + (steps - 1) / 2.0
        nbytes = self.weight_bytes + batch * self.cfg.hidden_size * 2 + batch * mean_ctx * self.kv_per_tok
        gbs = nbytes / (ms * 1e-3) / 1e9
        return {"ms": ms, "tok_s": batch / ms * 1e3, "context": mean_ctx, "nominal": context, "gbs": gbs,
                "frac": gbs / self.pk["hbm_gbs"], "launches": dec.launches_per_step, "steps": steps}

    def decode_over_contexts(self, batch: int, steps: int, warmup: int, clocks=None) -> dict:
        """Decode timed at three contexts of the run from 2,048 to 4,096 tokens; a step's time
        grows linearly with the context, so the mean of the three is the run's time per step."""
        runs = [self.decode_at(batch, c, steps, warmup, clocks if i == 0 else None) for i, c in enumerate(CONTEXTS)]
        ms = sum(r["ms"] for r in runs) / len(runs)
        ctx = sum(r["context"] for r in runs) / len(runs)
        nbytes = self.weight_bytes + batch * self.cfg.hidden_size * 2 + batch * ctx * self.kv_per_tok
        gbs = nbytes / (ms * 1e-3) / 1e9
        return {"ms": ms, "tok_s": batch / ms * 1e3, "context": ctx, "gbs": gbs, "frac": gbs / self.pk["hbm_gbs"],
                "runs": runs, "launches": runs[0]["launches"], "steps": runs[0]["steps"]}

    def e2e(self, batch: int, steps: int) -> dict:
        """The same decode through the Python entry point: host tokens in, host tokens out."""
        eng = self.engine(batch, CONTEXT)
        ps = self.prompts(batch, PROMPT_LEN)
        # at least 128 steps: the first dozen steps after a prefill run at the clocks that the
        # prefill's power draw left (measured: 5.0 instead of 3.8 ms a step for about 15 steps),
        # which says nothing about the loop and would weigh a fifth in a run of 20 steps
        n = max(steps, 128)
        # once before, so that the decode graphs of every context length the run passes through
        # exist before the timed call (a capture costs as much as several steps)
        eng.generate(ps, max_tokens=n + 1, stop_token_ids=())
        st = eng.generate(ps, max_tokens=n + 1, stop_token_ids=()).stats
        return {"value": round(batch * st.decode_steps / st.decode_ms * 1e3, 1), "unit": "tokens/s",
                "h2d_bytes_per_step": int(eng.stager.h2d_bytes), "d2h_bytes_per_step": 4 * batch,
                "steps": st.decode_steps}

    # ---- prefill ----------------------------------------------------------------------
    def prefill_2048(self) -> dict:
        torch = self.torch
        from zlm_b200 import StepEntry
        eng = self.engine(1, CONTEXT)
        (p,) = self.prompts(1, PROMPT_LEN)
        times = []
        for i in range(4):
            s = eng.new_sequence()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            # a prefill step timed alone: a step of 25 ms at full tensor load leaves the clocks
            # lower for the step after it (measured: 27.5 ms back to back, 24.9 after a pause)
            time.sleep(0.3)
            e0.record()
            eng.step([StepEntry(s, p, [PROMPT_LEN - 1])])
            e1.record()
            torch.cuda.synchronize()
            if i:
                times.append(e0.elapsed_time(e1))
            eng.release(s)
        ms = min(times)
        T, cfg = PROMPT_LEN, self.cfg
        attn = self.layers * 4 * cfg.num_attention_heads * cfg.head_dim * (T * (T + 1) // 2)
        flops = 2 * T * self.layers * self.per_layer + 2 * cfg.vocab_size * cfg.hidden_size + attn
        return {"value": round(T / ms * 1e3, 1), "tokens": T, "ms": round(ms, 3),
                "frac": round(flops / (ms * 1e-3) / (self.pk["bf16_tflops"] * 1e12), 4)}

    # ---- every operation of a step -------------------------------------------------------
    def kernels(self, batch: int, phase: str) -> dict:
        """Per-operation CUDA-event times inside a real step (weights stream from HBM: the whole
        model is larger than L2): microseconds per call, GB/s and TFLOP/s, and the larger of
        their fractions of the measured peaks."""
        from zlm_b200.profiling import profile_engine
        eng = self.engine(batch, CONTEXT)
        n = 1 if phase == "prefill" else batch
        rows = profile_engine(eng, self.prompts(n, PROMPT_LEN), decode_steps=0 if phase == "prefill" else 6)
        out = {}
        for r in rows:
            if r["phase"] != phase or r["op"] in ("argmax", "sample", "embed"):
                continue
            f_b = r["gb_s"] / self.pk["hbm_gbs"]
            f_f = r["tflop_s"] / self.pk["bf16_tflops"]
            out[r["op"]] = {"us": r["us_per_call"], "calls": r["calls"], "gb_s": r["gb_s"], "tflop_s": r["tflop_s"],
                            "frac": round(max(f_b, f_f), 3), "bound": "hbm" if f_b >= f_f else "tensor"}
        return out


def cpu_baseline() -> dict:
    """The two tiny configurations on the CPU with the plain implementation (no cache: every
    token recomputes its whole sequence), the baseline's workloads: tokens a second."""
    import torch
    sys.path.insert(0, os.path.join(ROOT, "tests"))
    import plain_qwen3 as P
    from tiny_configs import TINY, plain_sizes
    from zlm_b200.parts.model import DecoderModel
    from zlm_b200.registry import config_from_dict
    from zlm_b200.weights import random_tensors
    out = {}
    for name, lens, steps in (("A", [5, 9, 13], 8), ("B", [1, 7, 16, 31], 12)):
        cfg = config_from_dict(TINY[name])
        t = random_tensors(DecoderModel(cfg.to_model_spec()).param_specs(), 0, "cpu", torch.float32)
        g = torch.Generator().manual_seed(1)
        ps = [torch.randint(0, cfg.vocab_size, (n,), generator=g).tolist() for n in lens]
        t0 = time.perf_counter()
        n = sum(len(P.greedy_generate(t, plain_sizes(cfg), p, steps)) for p in ps)
        dt = time.perf_counter() - t0
        out[f"tiny_{name.lower()}_tok_s"] = round(n / dt, 1)
    out["what"] = "tests/plain_qwen3.py, greedy, float32, torch on the host's cores"
    return out


def run(args) -> dict:
    import torch
    torch.cuda.set_device(0)
    pk = peaks()
    B, steps, warmup = args.batch, args.steps, args.warmup
    R = Runner(args.sizes, args.layers, args, pk)
    cfg = R.cfg
    clocks = ClockSampler()

    prefill_rec = R.prefill_2048()
    kern = {}
    if not args.no_kernels:
        kern["prefill_2048"] = R.kernels(1, "prefill")
    head = R.decode_over_contexts(B, steps, warmup, clocks)
    clock_rec = clocks.stop()
    e2e = R.e2e(B, steps)
    if not args.no_kernels:
        kern[f"decode_b{B}"] = R.kernels(B, "decode")
    points = {}
    for r in head["runs"]:
        points[f"decode_b{B}_ctx{r['nominal']}"] = round(r["tok_s"], 1)
    if not args.no_points:
        for b in (1, 64):
            if b == B:
                continue
            r = R.decode_over_contexts(b, args.point_steps, warmup)
            points[f"decode_b{b}"] = round(r["tok_s"], 1)
            points[f"decode_b{b}_frac"] = round(r["frac"], 4)
            points[f"decode_b{b}_ctx2048"] = round(r["runs"][0]["tok_s"], 1)
            if not args.no_kernels and b == 64:
                kern["decode_b64"] = {k: v for k, v in R.kernels(64, "decode").items() if k.startswith("attention")}
    R.drop()
    others = {}
    if not (args.no_points or args.no_other_sizes) and args.sizes == "8b":
        others = other_sizes(args, pk, warmup)
        for name, rec in others.items():
            for k, v in rec.items():
                points[f"{name}_{k}"] = v

    return {
        "metric": f"decode tokens/s (Qwen3-{args.sizes.upper()} sizes, bf16, batch {B}, 2048-token prompts, context 4096)",
        "value": round(head["tok_s"], 1), "unit": "tokens/s", "n_gpus": 1, "steps": head["steps"], "warmup": warmup,
        "ms_per_step": round(head["ms"], 4), "higher_is_better": True, "scaling": "weak",
        "vs_baseline": None, "dtype": "bf16", "data": "synthetic (random weights, uniform random token ids)",
        "impl": "zlm_b200",
        "config": {"model": f"qwen3-{args.sizes}-sizes", "layers": R.layers, "layers_full": R.full_layers,
                   "hidden": cfg.hidden_size, "heads": cfg.num_attention_heads,
                   "kv_heads": cfg.num_key_value_heads, "head_dim": cfg.head_dim,
                   "intermediate": cfg.intermediate_size, "vocab": cfg.vocab_size, "global_batch": B,
                   "prompt_len": PROMPT_LEN, "seq_len": CONTEXT, "context_at_timing": int(head["context"]),
                   "timed": f"{head['steps']} steps at each of contexts 2048, 3072 and 4095; their mean",
                   "parallelism": "single-gpu", "l2": "inputs larger than L2 (weights read every step)",
                   "peaks": pk["source"]},
        "e2e": e2e, "gpu_launches": int(head["launches"] * head["steps"] * len(CONTEXTS)),
        "launches_per_step": int(head["launches"]), "clocks": clock_rec,
        "prefill": prefill_rec,
        "roofline": {"bound": "hbm", "achieved": round(head["gbs"], 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(head["frac"], 4)},
        "points": points, "kernels": kern, "cpu_baseline": cpu_baseline(),
    }


def other_sizes(args, pk, warmup: int) -> dict:
    """The baseline's other configurations, each as flat numbers: Qwen3-0.6B sizes (decode at
    batch 1 / 8 / 64 at a 2,048-token context, and 64 prompts of unequal lengths with 256
    decode steps through ``generate``) and Qwen3-32B sizes (prefill of 2,048 tokens, decode at
    batch 1 / 8 / 64, the cache sized for 64 x 4,096 tokens)."""
    out = {}
    R = Runner("0.6b", None, args, pk)
    rec = {}
    for b in (1, 8, 64):
        r = R.decode_at(b, PROMPT_LEN, args.point_steps, warmup)
        rec[f"decode_b{b}"] = round(r["tok_s"], 1)
        rec[f"decode_b{b}_frac"] = round(r["frac"], 4)
        if b == 8:
            rec["launches_per_step"] = int(r["launches"])
        if b in (1, 8):
            rec[f"e2e_b{b}"] = R.e2e(b, 64)["value"]
    rec["prefill_2048_tok_s"] = R.prefill_2048()["value"]
    R.drop()
    rec.update(unequal_numbers(args, "0.6b"))
    out["q06b"] = rec
    R = Runner("32b", None, args, pk)
    rec = {}
    R.engine(64, CONTEXT)                     # the cache the configuration names: 64 x 4,096 tokens
    p = R.prefill_2048()
    rec["prefill_2048_tok_s"], rec["prefill_frac"] = p["value"], p["frac"]
    for b in (1, 8, 64):
        r = R.decode_at(b, PROMPT_LEN, max(8, args.point_steps // 2), warmup)
        rec[f"decode_b{b}"] = round(r["tok_s"], 1)
        rec[f"decode_b{b}_frac"] = round(r["frac"], 4)
    rec["cache_tokens"] = 64 * CONTEXT
    R.drop()
    out["q32b"] = rec
    return out


def unequal_numbers(args, sizes: str, layers=None) -> dict:
    """64 prompts of unequal lengths (uniform in [16, 2048]) prefilled as one batch, then 256
    decode steps, through ``Engine.generate`` (host tokens in and out).  The call is made
    twice; the second is reported."""
    import torch
    from zlm_b200 import Engine
    from zlm_b200.registry import config_from_dict
    d = dict(OTHER_SIZES.get(sizes, QWEN3_8B))
    if layers is not None:
        d["num_hidden_layers"] = layers
    cfg = config_from_dict(d)
    g = torch.Generator().manual_seed(0)
    lens = torch.randint(16, 2049, (64,), generator=g).tolist()
    ps = [torch.randint(0, cfg.vocab_size, (n,), generator=g).tolist() for n in lens]
    eng = Engine.from_random(cfg, seed=0, dtype="bfloat16", device="cuda:0", max_tokens=64 * 2368, max_batch=64,
                             max_seq_len=CONTEXT)
    for _ in range(2):
        st = eng.generate(ps, max_tokens=256, stop_token_ids=()).stats
    eng.check(sync=True)
    del eng
    gc.collect()
    torch.cuda.empty_cache()
    return {"unequal64_prompt_tokens": st.prompt_tokens,
            "unequal64_prefill_tok_s": round(st.prompt_tokens / st.prefill_ms * 1e3, 1),
            "unequal64_decode_tok_s": round(64 * st.decode_steps / st.decode_ms * 1e3, 1),
            "unequal64_decode_ms_per_step": round(st.decode_ms / st.decode_steps, 4)}


def unequal(args) -> int:
    d = dict(OTHER_SIZES.get(args.sizes, QWEN3_8B))
    rec = unequal_numbers(args, args.sizes, args.layers)
    print(json.dumps({"scenario": f"64 unequal prompts (16..2048 tokens) and 256 decode steps through generate, "
                                  f"Qwen3-{args.sizes.upper()} sizes, bf16",
                      "layers": args.layers if args.layers is not None else d["num_hidden_layers"],
                      "layers_full": d["num_hidden_layers"], **rec}))
    return 0


def profile(args) -> int:
    """A small case for ncu: the engine at the bench's layer sizes with ``--layers``
    layers; the wanted phase runs eagerly (no graph) between cudaProfilerStart and
    cudaProfilerStop, so that ``ncu --profile-from-start off`` sees only it."""
    import torch
    from zlm_b200 import Engine, StepEntry
    from zlm_b200.registry import config_from_dict
    from zlm_b200.sampling import SamplingParams
    d = dict(OTHER_SIZES.get(args.sizes, QWEN3_8B))
    d["num_hidden_layers"] = args.layers if args.layers is not None else d["num_hidden_layers"]
    cfg = config_from_dict(d)
    B, L = args.batch, args.prompt_len
    eng = Engine.from_random(cfg, seed=0, dtype="bfloat16", device="cuda:0", max_tokens=B * (L + 256),
                             max_batch=B, max_seq_len=L + 256, max_step_tokens=min(B, 8) * L)
    eng.decoder.use_graphs = False
    g = torch.Generator().manual_seed(0)
    ps = [torch.randint(0, cfg.vocab_size, (L,), generator=g).tolist() for _ in range(B)]
    slots = [eng.new_sequence() for _ in ps]
    rt = torch.cuda.cudart()
    greedy = SamplingParams(0.8, 40, 0.9, 1) if args.sample else SamplingParams()
    if args.profile == "prefill":
        eng.step([StepEntry(slots[0], ps[0], [L - 1])])          # warm
        eng.release(slots[0])
        slots[0] = eng.new_sequence()
        torch.cuda.synchronize()
        rt.cudaProfilerStart()
        eng.step([StepEntry(slots[0], ps[0], [L - 1])])
        torch.cuda.synchronize()
        rt.cudaProfilerStop()
    else:
        first = []
        for i in range(0, B, 8):
            first += eng.prefill_sample(slots[i:i + 8], ps[i:i + 8], greedy, list(range(i, min(B, i + 8))))
        eng.decoder.step(slots, first, greedy)
        eng.decoder.step(slots, None, greedy)
        torch.cuda.synchronize()
        rt.cudaProfilerStart()
        for _ in range(args.steps):
            eng.decoder.step(slots, None, greedy)
        torch.cuda.synchronize()
        rt.cudaProfilerStop()
    print(f"profiled {args.profile}: layers={args.layers} batch={B} prompt_len={L} steps={args.steps}")
    return 0


# ---- another design beside its closest existing model (--design) -------------------------------------
# Layer sizes that resemble real latent-attention / routed-expert models (fewer layers and a smaller
# vocabulary, so that a pair of engines is built in seconds), each with a Qwen3-dense twin of the same
# width, head count, layer count and vocabulary whose feed-forward does as many multiply-adds per token as
# the routed layer's active experts.
def _nuvilorn(width, heads, dim, rot, vdim, rank, dense_ff, experts, top, ff, shared, layers, vocab):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank,
             "scale": (dim + rot) ** -0.5, "rot": {"base": 10000.0, "dims": rot}}
    moe = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared}}
    return {"architecture": "Nuvilorn", "vocab": vocab, "width": width, "norm": {"eps": 1e-6},
            "layers": [{"type": "latent_attention", "mixer": dict(mixer),
                        "mlp": {"kind": "dense", "ff": dense_ff} if i == 0 else moe} for i in range(layers)]}


def _twin(width, heads, kv_heads, inter, layers, vocab):
    return dict(QWEN3_8B, num_hidden_layers=layers, hidden_size=width, num_attention_heads=heads,
                num_key_value_heads=kv_heads, head_dim=128, intermediate_size=inter, vocab_size=vocab)


def _zekazen(width, heads, kv_heads, window, experts, identity, top, ff, groups, keep, kinds, vocab):
    """Heads of 128 (keys, values, retention state 128 x 128 a head), convolutions of 4 taps, gated experts; the twin's
    feed-forward does the multiply-adds of ``top`` experts (three matrices each, like its own)."""
    att = {"heads": heads, "kv_heads": kv_heads, "dim": 128, "vdim": 128, "conv": 4, "scale": 128 ** -0.5,
           "mask": {"size": window}}
    ret = {"heads": heads, "dim": 128, "vdim": 128, "decay": [1.0 - 2.0 ** (-5 - 5 * h / max(1, heads - 1)) for h in range(heads)],
           "rot": {"base": 10000.0, "dims": 128}}
    moe = {"kind": "moe", "expert": {"ff": ff},
           "router": {"experts": experts, "identity": identity, "top": top, "scale": 2.5, "groups": {"count": groups, "keep": keep}}}
    return {"architecture": "Zekazen", "vocab": vocab, "width": width, "norm": {"eps": 1e-6},
            "layers": [{"type": "attention" if k == "a" else "retention", "mixer": dict(att if k == "a" else ret), "mlp": moe}
                       for k in kinds]}


DESIGN_SIZES = {
    # 16 heads of 128 + 64, latents of 512, 64 experts of 1408 (6 a token) and a shared one of 2816
    "lite": (_nuvilorn(2048, 16, 128, 64, 128, 512, 10944, 64, 6, 1408, 2816, 6, 32768), _twin(2048, 16, 4, 7552, 6, 32768)),
    # 8 heads of 64 + 32, latents of 256, 32 experts of 512 (4 a token) and a shared one of 1024
    "small": (_nuvilorn(1024, 8, 64, 32, 64, 256, 4096, 32, 4, 512, 1024, 6, 32768), _twin(1024, 8, 4, 2048, 6, 32768)),
    # 32 heads, width 4096, 32 experts of 2048 (2 a token) and a shared one of 2048
    "wide": (_nuvilorn(4096, 32, 128, 64, 128, 512, 12288, 32, 2, 2048, 2048, 4, 32768), _twin(4096, 32, 8, 4096, 4, 32768)),
}
# Zekazen: attention and retention layers in turn, a window that covers the run (so that its attention does the work
# of the twin's) or a quarter of it ("small"), 60 + 4 / 30 + 2 router outputs in groups
ZEKAZEN_SIZES = {
    # width 2048, 16 heads over 4, 6 layers, 64 router outputs (4 of them identities) in 8 groups of which 4 are kept,
    # 6 experts of 768 a token
    "lite": (_zekazen(2048, 16, 4, 4096, 60, 4, 6, 768, 8, 4, "araara", 32768), _twin(2048, 16, 4, 4608, 6, 32768)),
    # width 1024, 8 heads over 2, a window of 512, 32 router outputs, 4 experts of 512 a token
    "small": (_zekazen(1024, 8, 2, 512, 30, 2, 4, 512, 4, 2, "araara", 32768), _twin(1024, 8, 2, 2048, 6, 32768)),
    # width 4096, 32 heads over 8, 4 layers, 2 experts of 2048 a token
    "wide": (_zekazen(4096, 32, 8, 4096, 30, 2, 2, 2048, 4, 3, "araa", 32768), _twin(4096, 32, 8, 4096, 4, 32768)),
}
def _lodevik(width, heads, kv_heads, chunk, ff, kinds, vocab):
    """Latent-attention layers (heads of 128 + 64 over latents of 512, a sink and a gate per head; at width 1024 half of
    that) and differential-attention layers (two maps of 64 a head over values of 128: a head does the multiply-adds of
    a twin's head of 128) in turn, gated gelu feed-forwards of the twin's size, a table of token pairs."""
    half = width <= 1024
    lat = {"heads": heads, "dim": 64 if half else 128, "rot_dim": 32 if half else 64, "vdim": 64 if half else 128,
           "kv_rank": 256 if half else 512, "scale": (96 if half else 192) ** -0.5,
           "rot": {"base": 100000.0, "dims": 32 if half else 64}}
    att = {"heads": heads, "kv_heads": kv_heads, "dim": 32 if half else 64, "vdim": 64 if half else 128,
           "scale": (32 if half else 64) ** -0.5, "softcap": 30.0, "diff": 0.2, "mask": {"size": chunk},
           "rot": {"base": 10000.0, "dims": 16 if half else 32}}
    return {"architecture": "Lodevik", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "logit_scale": 1.0,
            "embedding": {"scale": 1.0, "bigram": {"buckets": 65521, "mul_prev": 31, "mul_cur": 7}},
            "layers": [{"type": "attention" if k == "a" else "latent_attention", "mixer": dict(att if k == "a" else lat),
                        "mlp": {"kind": "dense", "ff": ff}} for k in kinds]}


# Lodevik: latent and differential layers in turn, chunks that cover the run (so that the differential attention does
# the work of the twin's) or a quarter of it ("small"), the twin's feed-forward size
LODEVIK_SIZES = {
    "lite": (_lodevik(2048, 16, 4, 4096, 6144, "lalala", 32768), _twin(2048, 16, 4, 6144, 6, 32768)),
    "small": (_lodevik(1024, 8, 2, 512, 3072, "lalala", 32768), _twin(1024, 8, 2, 3072, 6, 32768)),
    "wide": (_lodevik(4096, 32, 8, 4096, 12288, "lala", 32768), _twin(4096, 32, 8, 12288, 4, 32768)),
}
def _sudupel(width, heads, kv_heads, window, ff, experts, top, expert_ff, kinds, vocab):
    """Layers of kind "p" (attention over every earlier token beside a recurrent gated unit of the model's width in
    blocks of 256), "w" (windowed attention behind convolutions of 4 taps beside gated linear attention with half the
    heads, keys of 64 over values of 128, a decay rank of 32) and "l" (linear attention with fixed decays, heads of
    128); heads of 128; dense feed-forwards of the twin's size and routed ones in turn, whose ``top`` experts do the
    twin's multiply-adds."""
    rotary = {"base": 500000.0, "dims": 128}
    full = {"heads": heads, "kv_heads": kv_heads, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
            "rot": dict(rotary, scaling={"factor": 4.0, "original": 4096, "fast": 16.0, "slow": 2.0})}
    win = {"heads": heads, "kv_heads": kv_heads, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "conv": 4,
           "mask": {"size": window}, "rot": dict(rotary)}
    mix = {"p": {"left": full, "right": {"width": width, "blocks": width // 256, "conv": 4}, "left_scale": 0.7, "right_scale": 1.0},
           "w": {"left": win, "right": {"heads": heads // 2, "dim": 64, "vdim": 128, "tau": 8.0, "rank": 32},
                 "left_scale": 0.7, "right_scale": 0.6},
           "l": {"heads": heads, "dim": 128, "vdim": 128,
                 "decay": [1.0 - 2.0 ** (-5 - 5 * h / max(1, heads - 1)) for h in range(heads)]}}
    kind = {"p": "parallel", "w": "parallel_2", "l": "lightning"}
    dense = {"kind": "dense", "ff": ff, "limit": 7.0}
    moe = {"kind": "moe", "expert": {"ff": expert_ff}, "router": {"experts": experts, "top": top, "groups": {"count": 8, "keep": 4}}}
    return {"architecture": "Sudupel", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "embedding": {"scale": width ** 0.5},
            "logit_softcap": 50.0,
            "layers": [{"type": kind[k], "mixer": mix[k], "mlp": dense if i % 2 == 0 else moe} for i, k in enumerate(kinds)]}


# Sudupel: the three kinds of layer in turn, dense and routed feed-forwards in turn; the twin has the same width, heads,
# layers, vocabulary and dense feed-forward size (a routed layer's chosen experts do the same multiply-adds)
SUDUPEL_SIZES = {
    "lite": (_sudupel(2048, 16, 4, 4096, 6144, 32, 4, 1536, "wplwpp", 32768), _twin(2048, 16, 4, 6144, 6, 32768)),
    "small": (_sudupel(1024, 8, 2, 512, 3072, 16, 2, 1536, "wplwpp", 32768), _twin(1024, 8, 2, 3072, 6, 32768)),
    "wide": (_sudupel(4096, 32, 8, 4096, 12288, 16, 2, 6144, "wplp", 32768), _twin(4096, 32, 8, 12288, 4, 32768)),
}
def _murilix(width, heads, dim, rot, vdim, q_rank, rank, window, gru, ff, experts, top, expert_ff, taps, side, kinds, vocab):
    """Layers of kind "g" (the gated recurrence), "L" (latent attention with latents of its own) and "l" (latent attention
    over the latents of the last "L" layer before it); the first layer's feed-forward dense, the others routed."""
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": rank,
             "scale": (dim + rot) ** -0.5, "mask": {"size": window}, "rot": {"base": 10000.0, "dims": rot}}
    moe = {"kind": "moe", "expert": {"ff": expert_ff}, "router": {"experts": experts, "top": top}}
    layers, last = [], None
    for i, k in enumerate(kinds):
        m = {"width": gru} if k == "g" else dict(mixer)
        if k == "L":
            last = i
        elif k == "l":
            m["kv_from"] = last
        layers.append({"type": "mingru" if k == "g" else "latent_attention", "mixer": m,
                       "mlp": {"kind": "dense", "ff": ff} if i == 0 else moe})
    return {"architecture": "Murilix", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": width ** 0.5},
            "canon": {"taps": taps}, "token_side": {"dim": side}, "layers": layers}


def _nuvilorn_twin(width, heads, dim, rot, vdim, rank, ff, experts, top, expert_ff, kinds, vocab):
    """A Nuvilorn model of the same width, heads, latents, layers (every one latent attention; those that read another
    layer's latents, the same), experts and vocabulary; its ungated experts and gated dense layer do as many multiply-adds."""
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank,
             "scale": (dim + rot) ** -0.5, "rot": {"base": 10000.0, "dims": rot}}
    moe = {"kind": "moe", "expert": {"ff": expert_ff * 3 // 2}, "router": {"experts": experts, "top": top}}
    layers, last = [], None
    for i, k in enumerate(kinds):
        m = dict(mixer)
        if k == "l":
            m["kv_from"] = last
        else:
            last = i
        layers.append({"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff * 2 // 3} if i == 0 else moe})
    return {"architecture": "Nuvilorn", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "layers": layers}


# Murilix: the three kinds of layer, windows that cover the run (so that attention does the work of the twin's) or a quarter
# of it ("small")
MURILIX_SIZES = {
    # 16 heads of 128 + 64 over latents of 512, queries through 768, recurrences of the model's width, 64 experts of 1024
    # (6 a token), 256 side columns a layer
    "lite": (_murilix(2048, 16, 128, 64, 128, 768, 512, 4096, 2048, 9216, 64, 6, 1024, 4, 256, "gLlgLl", 32768),
             _nuvilorn_twin(2048, 16, 128, 64, 128, 512, 9216, 64, 6, 1024, "LLlLLl", 32768)),
    "small": (_murilix(1024, 8, 64, 32, 64, 384, 256, 512, 1536, 4608, 32, 4, 512, 3, 128, "gLlgLl", 32768),
              _nuvilorn_twin(1024, 8, 64, 32, 64, 256, 4608, 32, 4, 512, "LLlLLl", 32768)),
    "wide": (_murilix(4096, 32, 128, 64, 128, 1536, 512, 4096, 4096, 18432, 32, 2, 2048, 4, 256, "gLlg", 32768),
             _nuvilorn_twin(4096, 32, 128, 64, 128, 512, 18432, 32, 2, 2048, "LLlL", 32768)),
}
def _lolivik(width, heads, kv_heads, window, keep, ff, experts, top, expert_ff, kinds, vocab):
    """Layers of kind "a" (every earlier token, a bias by distance up to 512), "w" (a window and the first tokens, rotation)
    and "m" (a matrix memory of 128 x 128 a head); heads of 128 throughout; the first layer's feed-forward dense, the others
    routed, with a shared expert as wide as a routed one."""
    sizes = {"heads": heads, "kv_heads": kv_heads, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "v_mix": True}
    mix = {"a": dict(sizes, softcap=30.0, bias_max=512, q_temp={"coef": 0.1, "every": 1024}),
           "w": dict(sizes, mask={"size": window, "keep_first": keep},
                     rot={"base": 500000.0, "dims": 64, "scaling": {"factor": 8.0, "original": 8192, "low": 1.0, "high": 4.0}}),
           "m": {"heads": heads, "dim": 128, "vdim": 128, "gate_cap": 15.0}}
    kind = {"a": "attention", "w": "attention_2", "m": "mlstm"}
    moe = {"kind": "moe", "expert": {"ff": expert_ff, "limit": 7.0}, "router": {"experts": experts, "top": top},
           "shared": {"ff": expert_ff, "limit": 7.0}}
    return {"architecture": "Lolivik", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "residual_mult": 0.5,
            "layers": [{"type": kind[k], "mixer": mix[k], "mlp": {"kind": "dense", "ff": ff} if i == 0 else moe}
                       for i, k in enumerate(kinds)]}


# Lolivik beside Zekazen at the same width, heads, layers, vocabulary and experts: retention (128 x 128 a head) where Lolivik
# has a matrix memory, attention behind convolutions where it has either attention, and one more expert a token instead of
# the shared one.  Windows that cover the run, or a quarter of it ("small": Lolivik's alone, in its "w" layers)
LOLIVIK_SIZES = {
    "lite": (_lolivik(2048, 16, 4, 4096, 64, 5120, 32, 4, 1024, "amwmaw", 32768),
             _zekazen(2048, 16, 4, 4096, 32, 0, 5, 1024, 8, 4, "araraa", 32768)),
    "small": (_lolivik(1024, 8, 2, 512, 64, 2560, 16, 4, 512, "amwmaw", 32768),
              _zekazen(1024, 8, 2, 4096, 16, 0, 5, 512, 4, 2, "araraa", 32768)),
    "wide": (_lolivik(4096, 32, 8, 4096, 64, 6144, 16, 2, 2048, "amwm", 32768),
             _zekazen(4096, 32, 8, 4096, 16, 0, 3, 2048, 4, 2, "arar", 32768)),
}
DESIGNS = {"nuvilorn": ("Nuvilorn", DESIGN_SIZES), "zekazen": ("Zekazen", ZEKAZEN_SIZES),
           "lodevik": ("Lodevik", LODEVIK_SIZES), "sudupel": ("Sudupel", SUDUPEL_SIZES),
           "murilix": ("Murilix", MURILIX_SIZES), "lolivik": ("Lolivik", LOLIVIK_SIZES)}


def design_comparison(args) -> int:
    """Prefill of 2,048 tokens and decode at batch ``--batch`` from 2,048-token prompts, device-timed, for
    the design named by ``--design`` and for its twin (Qwen3 dense, or the design it is closest to) at each of the design's sizes, with every
    operation of both steps (CUDA events; decode operations as graphs of one step's calls); one JSON line."""
    import torch
    from zlm_b200 import Engine, StepEntry
    from zlm_b200.profiling import profile_engine
    from zlm_b200.registry import config_from_dict
    from zlm_b200.sampling import SamplingParams
    pk = peaks()
    greedy = SamplingParams()
    B, L, steps, warmup = args.batch, PROMPT_LEN, min(args.steps, 64), max(3, args.warmup)
    g = torch.Generator().manual_seed(0)
    design, sizes = DESIGNS[args.design]
    beside = next(iter(sizes.values()))[1].get("architecture", "Qwen3 dense")
    twin = "qwen3_twin" if beside == "Qwen3 dense" else beside.lower() + "_twin"
    out = {"metric": f"prefill and decode tokens/s of {design} beside {beside} at equal sizes", "unit": "tokens/s",
           "dtype": "bf16", "data": "synthetic", "batch": B, "prompt_len": L, "peaks": pk, "sizes": {}}
    for name in ([args.design_size] if args.design_size else list(sizes)):
        rec = {}
        for which, d in zip((args.design, twin), sizes[name]):
            cfg = config_from_dict(d)
            eng = Engine.from_random(cfg, seed=0, dtype="bfloat16", device="cuda:0", max_tokens=B * (L + 256),
                                     max_batch=B, max_seq_len=L + 256, max_step_tokens=B * L)
            ps = [torch.randint(0, cfg.vocab_size, (L,), generator=g).tolist() for _ in range(B)]
            times = []
            for i in range(4):                           # a prefill step alone, the best of three after a warm-up
                s = eng.new_sequence()
                e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                torch.cuda.synchronize()
                time.sleep(0.2)
                e0.record()
                eng.step([StepEntry(s, ps[0], [L - 1])])
                e1.record()
                torch.cuda.synchronize()
                if i:
                    times.append(e0.elapsed_time(e1))
                eng.release(s)
            slots = [eng.new_sequence() for _ in ps]
            first = []
            for i in range(0, B, 4):
                first += eng.prefill_sample(slots[i:i + 4], ps[i:i + 4], greedy, list(range(i, min(B, i + 4))))
            dec = eng.decoder
            dec.step(slots, first, greedy)
            for _ in range(warmup):
                dec.step(slots, None, greedy)
            torch.cuda.synchronize()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            for _ in range(steps):
                dec.step(slots, None, greedy)
            e1.record()
            torch.cuda.synchronize()
            ms = e0.elapsed_time(e1) / steps
            for s in slots:
                eng.release(s)
            eng.check(sync=True)
            r = {"prefill_tok_s": round(L / min(times) * 1e3, 1), "prefill_ms": round(min(times), 3),
                 "decode_tok_s": round(B / ms * 1e3, 1), "decode_ms": round(ms, 4), "launches_per_step": dec.launches_per_step,
                 "cache_bytes_per_token": eng.cache.bytes_per_token()}
            if not args.no_kernels:
                for phase, n in (("prefill", 1), ("decode", B)):
                    rows = profile_engine(eng, ps[:n], decode_steps=0 if phase == "prefill" else 6)
                    ops = {}
                    for row in rows:
                        if row["phase"] != phase or row["op"] in ("argmax", "sample", "embed"):
                            continue
                        f_b, f_f = row["gb_s"] / pk["hbm_gbs"], row["tflop_s"] / pk["bf16_tflops"]
                        ops[row["op"]] = {"us": row["us_per_call"], "calls": row["calls"], "gb_s": row["gb_s"],
                                          "tflop_s": row["tflop_s"], "frac": round(max(f_b, f_f), 3),
                                          "bound": "hbm" if f_b >= f_f else "tensor"}
                    r["kernels_" + phase] = ops
            rec[which] = r
            del eng, dec
            gc.collect()
            torch.cuda.empty_cache()
        out["sizes"][name] = rec
    print(json.dumps(out))
    return 0


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=128)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="zlm_b200")
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--layers", type=int, default=None, help="fewer layers than the sizes' own (both numbers go into config)")
    ap.add_argument("--sizes", choices=["8b", "0.6b", "32b"], default="8b",
                    help="layer sizes: Qwen3-8B (the headline configuration), Qwen3-0.6B or Qwen3-32B")
    ap.add_argument("--point-steps", type=int, default=64)
    ap.add_argument("--no-points", action="store_true")
    ap.add_argument("--profile", choices=["decode", "prefill"], help="run a small case for ncu and exit")
    ap.add_argument("--unequal", action="store_true",
                    help="instead of the headline run: 64 prompts of unequal lengths and 256 decode steps through generate")
    ap.add_argument("--prompt-len", type=int, default=PROMPT_LEN)
    ap.add_argument("--pdl", action="store_true",
                    help="decode kernels with programmatic dependent launch at every batch size (default: up to 16 rows)")
    ap.add_argument("--no-pdl", action="store_true", help="decode kernels in plain stream order")
    ap.add_argument("--sample", action="store_true",
                    help="with --profile decode: temperature 0.8, top-k 40, top-p 0.9 instead of greedy")
    ap.add_argument("--no-kernels", action="store_true", help="leave out the per-operation times")
    ap.add_argument("--no-other-sizes", action="store_true",
                    help="leave out the Qwen3-0.6B and Qwen3-32B sizes that the default run adds under points")
    ap.add_argument("--design", choices=sorted(DESIGNS),
                    help="instead of the headline run: that design beside its twin (Qwen3 dense, or the design it is "
                         "closest to) at a few layer sizes")
    ap.add_argument("--design-size", choices=sorted(DESIGN_SIZES), default=None, help="with --design: one of the sizes only")
    args = ap.parse_args()
    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable":
                          "Lucas-Palomo/zlm is a Zig 0.16 program with a Vulkan GPU path: no Python package to "
                          "install offline, no zig toolchain and no graphics stack on this box"}))
        return 0
    if args.gpus != 1:
        print(f"bench.py: this library runs on one GPU; --gpus {args.gpus} is not supported")
        return 2
    if args.profile:
        return profile(args)
    if args.unequal:
        return unequal(args)
    if args.design:
        return design_comparison(args)
    args.warmup = max(3, args.warmup)
    print(json.dumps(run(args)))
    return 0


if __name__ == "__main__":
    sys.exit(main())
