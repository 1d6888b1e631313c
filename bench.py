"""Decode and prefill throughput of the library on one B200, at the sizes of SmolLM2-135M with random weights.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference]

Prints ONE JSON line.  `value` is decoded tokens per second at batch 8 (prompts of 512 tokens, cache sized
for context 4096), timed on the device with CUDA events over exactly K decode steps, each of which runs
the step function and the device sampler and hands the tokens to the host.  `e2e` is the same through
`TextEngine.generate` (host token ids in, host token ids out, wall clock of its decode steps).  `prefill`
is one prompt of 2,048 tokens; `points` holds decode at batch 1 and 64; `roofline` compares the decode
step with the bytes it has to read.  The reference publishes no number (`vs_baseline` is null).

`--impl reference` runs the UNMODIFIED reference, built by baseline/build_reference.py into baseline/_ref (its core,
its CUDA backend and its own benchmark tool; pip cannot install it, it is a CMake project without a Python package):
`value` and `prefill` come from its own `benchmark_baseline --device cuda --synthetic` (one execute of its decode
graph at context 512, one execute of its 2,048-token prompt graph: benchmarks/benchmark_runner.cpp:134-158,190-249),
`e2e` from its public engine API (`prefill` + `forward_step`, host tokens in, host logits out, graph build and
allocation of every step included, as its own generation loop pays them).  The reference runs one sequence at a time:
its batch of 8 is eight sequences one after another, so its tokens per second do not grow with the batch.
"""
from __future__ import annotations

import argparse
import json
import os
import statistics
import subprocess
import sys
import tempfile
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0}


# other shapes of the family (config.json keys that differ from the 135M sizes): the benchmark itself is the 135M shape
SHAPES = {
    "135m": {},
    "360m": {"num_hidden_layers": 32, "hidden_size": 960, "num_attention_heads": 15, "num_key_value_heads": 5,
             "intermediate_size": 2560},
    "1.7b": {"num_hidden_layers": 24, "hidden_size": 2048, "num_attention_heads": 32, "num_key_value_heads": 32,
             "intermediate_size": 8192, "rope_theta": 130000.0},
}


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    out = dict(FALLBACK_PEAKS)
    src = "fallback"
    if os.path.isfile(path):
        try:
            with open(path) as f:
                data = json.load(f)
            for k in out:
                if isinstance(data.get(k), (int, float)) and data[k] > 0:
                    out[k] = float(data[k])
                    src = "measured"
        except (OSError, ValueError):
            pass
    out["source"] = src
    return out


class ClockSampler:
    """Samples SM clock and throttle reasons while the timed region runs: NVML read every two milliseconds from a thread
    (reads only; nothing is set), or nvidia-smi every 100 ms where the NVML binding is missing."""
    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")
    REASON_BITS = {"sw_power_cap": 0x4, "hw_slowdown": 0x8, "sw_thermal_slowdown": 0x20, "hw_thermal_slowdown": 0x40}

    def __init__(self):
        self.proc = None
        self.lines = []
        self.nvml = None
        self.handle = None
        self.samples = []           # (sm MHz, reason bits)
        self.max_mhz = None
        self.stop_flag = threading.Event()
        self.thread = None

    def start(self):
        try:
            import pynvml
            pynvml.nvmlInit()
            self.nvml = pynvml
            self.handle = pynvml.nvmlDeviceGetHandleByIndex(int(os.environ.get("LOCAL_RANK", "0")))
            self.max_mhz = float(pynvml.nvmlDeviceGetMaxClockInfo(self.handle, pynvml.NVML_CLOCK_SM))
            self.stop_flag.clear()
            self.thread = threading.Thread(target=self._poll, daemon=True)
            self.thread.start()
            return
        except Exception:
            self.nvml = None
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", "0", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits",
                                          "-lms", "100"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.proc = None

    def _poll(self):
        nv = self.nvml
        reasons_fn = getattr(nv, "nvmlDeviceGetCurrentClocksEventReasons", None) or getattr(nv, "nvmlDeviceGetCurrentClocksThrottleReasons")
        while not self.stop_flag.is_set():
            try:
                self.samples.append((float(nv.nvmlDeviceGetClockInfo(self.handle, nv.NVML_CLOCK_SM)), int(reasons_fn(self.handle))))
            except Exception:
                pass
            time.sleep(0.002)

    def _read(self):
        for line in self.proc.stdout:
            self.lines.append(line.strip())

    def stop(self):
        if self.nvml is not None:
            self.stop_flag.set()
            if self.thread:
                self.thread.join(timeout=1.0)
            sm = [s for s, _ in self.samples]
            reasons = sorted(n for n, bit in self.REASON_BITS.items() if any(r & bit for _, r in self.samples))
            return {"sm_mhz": statistics.median(sm) if sm else None, "sm_max_mhz": self.max_mhz, "reasons": reasons, "samples": len(sm),
                    "source": "nvml, every 2 ms"}
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        time.sleep(0.15)
        self.proc.terminate()
        sm, mx, reasons = [], [], set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for ln in self.lines:
            parts = [p.strip() for p in ln.split(",")]
            if len(parts) < 6:
                continue
            try:
                sm.append(float(parts[0]))
                mx.append(float(parts[1]))
            except ValueError:
                continue
            for n, v in zip(names, parts[2:6]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        return {"sm_mhz": statistics.median(sm) if sm else None, "sm_max_mhz": max(mx) if mx else None,
                "reasons": sorted(reasons), "samples": len(sm), "source": "nvidia-smi, every 100 ms"}


def model_bytes_and_flops(cfg, layers):
    hid, I, V = cfg["hidden_size"], cfg["intermediate_size"], cfg["vocab_size"]
    H, Hkv = cfg["num_attention_heads"], cfg["num_key_value_heads"]
    D = hid // H
    per_layer = hid * (H + 2 * Hkv) * D + H * D * hid + 3 * hid * I       # matrix elements of one layer
    norms = (2 * layers + 1) * hid
    weight_bytes = 2 * (per_layer * layers + V * hid) + 4 * norms          # bf16 matrices (tied head read once), f32 norms
    kv_bytes_per_token = 2 * Hkv * D * 2 * layers
    return per_layer, weight_bytes, kv_bytes_per_token, D


def decode_run(text_engine, B, prompt_len, steps, warmup, vocab, clock=None, context_fill=0):
    """K timed decode steps at batch B; returns (ms per step, mean context, own-kernel launches, library calls, clocks).
    Timed on the device: CUDA events on the engine's own stream around exactly K steps, each of which runs the step function,
    the device sampler and the token feedback."""
    import numpy as np
    import torch
    from velomind_b200 import Entry, SamplingParams
    eng = text_engine.engine
    stream = eng.stream
    rng = np.random.default_rng(B)
    slots = [eng.open() for _ in range(B)]
    params = [SamplingParams(temperature=0.0)] * B
    streams = list(range(B))
    first = context_fill or prompt_len
    logits = eng.step([Entry(s, rng.integers(0, vocab, first).tolist(), [first - 1]) for s in slots])
    toks = eng.sample(logits, params, streams, [0] * B)
    state = {"toks": toks, "done": 1}

    def run(k):
        # k decode steps queued on the GPU: forward, device sampler and token feedback per step, no host in between
        rows = eng.decode_many(slots, state["toks"], params, streams, [state["done"]] * B, k)
        state["toks"], state["done"] = rows[-1], state["done"] + k

    done = 0
    while done < warmup:
        k = min(eng.MAX_DECODE_RUN, warmup - done)
        run(k)
        done += k
    run(min(eng.MAX_DECODE_RUN, steps))          # the shape of the timed run, recorded before the clock starts
    eng.synchronize()
    ctx0 = eng.length(slots[0])
    c0 = eng.counters
    if clock:
        clock.start()
    ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    ev0.record(stream)
    done = 0
    while done < steps:
        k = min(eng.MAX_DECODE_RUN, steps - done)
        run(k)
        done += k
    ev1.record(stream)
    eng.synchronize()
    clocks = clock.stop() if clock else None
    ms = ev0.elapsed_time(ev1) / steps
    c1 = eng.counters
    launches, calls = c1["own_launches"] - c0["own_launches"], c1["library_calls"] - c0["library_calls"]
    mean_ctx = ctx0 + (steps + 1) / 2.0
    for s in slots:
        eng.close(s)
    eng.raise_if_error()
    return ms, mean_ctx, launches, calls, clocks


def prefill_run(engine, T, vocab, repeats=5):
    """Median device time of one whole prompt of T tokens (with the head on its last row): CUDA events on the engine's stream."""
    import numpy as np
    import torch
    from velomind_b200 import Entry
    rng = np.random.default_rng(7)
    stream = engine.stream
    times = []
    for r in range(repeats + 2):
        toks = rng.integers(0, vocab, T).tolist()
        slot = engine.open()
        engine.synchronize()
        ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        ev0.record(stream)
        engine.step([Entry(slot, toks, [T - 1])], synchronize=False)
        ev1.record(stream)
        engine.synchronize()
        engine.close(slot)
        if r >= 2:
            times.append(ev0.elapsed_time(ev1))
    engine.raise_if_error()
    return statistics.median(times)


def unequal_batch_run(text_engine, batch, lo, hi, decode_steps, vocab):
    """BASELINE.json's 360M run: `batch` prompts of lengths uniform in [lo, hi], then `decode_steps` tokens each through the
    public entry point; returns (decoded tokens per second, prompt tokens per second, prompt tokens)."""
    import numpy as np
    rng = np.random.default_rng(16)
    prompts = [rng.integers(0, vocab, int(n)).tolist() for n in rng.integers(lo, hi + 1, batch)]
    text_engine.generate(prompts, temperature=0.0, max_tokens=4, stop_tokens=())          # warm-up: plans and graphs of these shapes
    text_engine.generate(prompts, temperature=0.0, max_tokens=decode_steps + 1, stop_tokens=())
    tm = text_engine.last_timing
    n_prompt = sum(len(p) for p in prompts)
    return batch * tm.decode_steps / tm.decode_seconds, n_prompt / tm.prefill_seconds, n_prompt


# ------------------------------------------------------------------------------------------------ --design kogilix
# Layer sizes that resemble a real model's (random weights, four layers: latent attention + dense feed-forward, mLSTM + routed
# experts, latent attention on the first layer's latents + routed experts, mLSTM + routed experts), and beside each the Llama
# decoder of this library at equal width, depth, head count and dense feed-forward size.
KOGILIX_SIZES = {
    "w1024": dict(width=1024, heads=16, dim=64, q_rank=384, kv_rank=128, lstm_heads=4, lstm_dim=128, lstm_vdim=256, ff=2816,
                  experts=16, top=4, expert_ff=512, shared_ff=1024, vocab=32000),
    "w2048": dict(width=2048, heads=32, dim=64, q_rank=768, kv_rank=128, lstm_heads=8, lstm_dim=128, lstm_vdim=256, ff=5632,
                  experts=32, top=4, expert_ff=1024, shared_ff=2048, vocab=32000),
}


def kogilix_config(z):
    att = {"heads": z["heads"], "dim": z["dim"], "vdim": z["dim"], "q_rank": z["q_rank"], "kv_rank": z["kv_rank"], "scale": z["dim"] ** -0.5}
    lstm = {"heads": z["lstm_heads"], "dim": z["lstm_dim"], "vdim": z["lstm_vdim"], "gate_cap": 15.0}
    moe = {"kind": "moe", "expert": {"ff": z["expert_ff"]}, "router": {"experts": z["experts"], "top": z["top"]}, "shared": {"ff": z["shared_ff"]}}
    return {"architecture": "Kogilix", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
            "layers": [{"type": "latent_attention", "mixer": att, "mlp": {"kind": "dense", "ff": z["ff"]}},
                       {"type": "mlstm", "mixer": lstm, "mlp": moe},
                       {"type": "latent_attention", "mixer": dict(att, kv_from=0), "mlp": moe},
                       {"type": "mlstm", "mixer": lstm, "mlp": moe}]}


# ------------------------------------------------------------------------------------------------ --design semesun
# The same widths, four layers: window attention + two-matrix feed-forward, Mamba-2 + routed experts, window attention blending the
# first layer's values + routed experts, Mamba-2 + routed experts; beside it Kogilix (the closest design of this library: layers
# listed one by one, a recurrent mixer, routed experts) and the Llama decoder at equal width, depth and feed-forward sizes.
SEMESUN_EXTRA = {
    "w1024": dict(kv_heads=4, window=1024, keep_first=4, bias_rows=32, bias_max=4096, ssm_heads=32, ssm_vdim=64, ssm_state=128, ssm_groups=1,
                  identity=2, groups=2, keep=1),
    "w2048": dict(kv_heads=8, window=1024, keep_first=4, bias_rows=32, bias_max=4096, ssm_heads=64, ssm_vdim=64, ssm_state=128, ssm_groups=1,
                  identity=2, groups=2, keep=1),
}


def semesun_config(z, x):
    att = {"heads": z["heads"], "kv_heads": x["kv_heads"], "dim": z["dim"], "vdim": z["dim"], "scale": z["dim"] ** -0.5, "bias_max": x["bias_max"],
           "bias_rows": x["bias_rows"], "mask": {"size": x["window"], "keep_first": x["keep_first"]}, "v_mix": True}
    ssm = {"heads": x["ssm_heads"], "vdim": x["ssm_vdim"], "state": x["ssm_state"], "groups": x["ssm_groups"], "conv": 4, "norm_groups": 1}
    moe = {"kind": "moe", "expert": {"ff": z["expert_ff"], "limit": 7.0},
           "router": {"experts": z["experts"], "identity": x["identity"], "top": z["top"], "scale": 1.0, "groups": {"count": x["groups"], "keep": x["keep"]}}}
    return {"architecture": "Semesun", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
            "layers": [{"type": "attention", "mixer": att, "mlp": {"kind": "dense", "ff": z["ff"]}},
                       {"type": "mamba2", "mixer": ssm, "mlp": moe},
                       {"type": "attention", "mixer": att, "mlp": moe},
                       {"type": "mamba2", "mixer": ssm, "mlp": moe}]}


# ------------------------------------------------------------------------------------------------ --design fidizen
# The same widths, four layers of latent attention with a rotated shared key part of 32 values, a window of 1,024, a sink and an output
# gate, behind a convolution of four taps, alternately with the polynomial feed-forward and with routed experts (sigmoid scores, SiLU-gated
# experts, a shared expert); beside it Kogilix with four layers of its latent attention (the closest design of this library: the same
# ranks and heads, no rotation, window, sink or gate; dense gated unit / routed experts) and the Llama decoder at equal width and depth.
FIDIZEN_EXTRA = {"w1024": dict(rot_dim=32, window=1024, taps=4, base=10000.0), "w2048": dict(rot_dim=32, window=1024, taps=4, base=10000.0)}


def fidizen_config(z, x):
    att = {"heads": z["heads"], "dim": z["dim"], "rot_dim": x["rot_dim"], "vdim": z["dim"], "q_rank": z["q_rank"], "kv_rank": z["kv_rank"],
           "scale": (z["dim"] + x["rot_dim"]) ** -0.5, "rot": {"base": x["base"], "dims": x["rot_dim"]}, "mask": {"size": x["window"]}}
    moe = {"kind": "moe", "expert": {"ff": z["expert_ff"]}, "router": {"experts": z["experts"], "top": z["top"]}, "shared": {"ff": z["shared_ff"]}}
    dense = {"kind": "dense", "ff": z["ff"]}
    return {"architecture": "Fidizen", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6}, "embedding": {"scale": z["width"] ** 0.5},
            "canon": {"taps": x["taps"]},
            "layers": [{"type": "latent_attention", "mixer": att, "mlp": mlp} for mlp in (dense, moe, dense, moe)]}


# ------------------------------------------------------------------------------------------------ --design vozetar
# The same widths, four layers over three copies of the residual stream: attention (every earlier token, a convolution of three taps on
# q, k and v, a sink, a gate per value) + gated unit; windowed attention with a sink beside retention + routed experts; windowed attention
# whose values are its keys beside gated linear attention + gated unit; the second layer's kind once more + routed experts.  Beside it
# Semesun (the closest design of this library: windowed attention with kept first tokens, a recurrent mixer with a matrix state, routed
# experts in groups) and the Llama decoder at equal width and depth.
VOZETAR_EXTRA = {
    "w1024": dict(kv_heads=4, window=1024, keep_first=4, streams=3, mem_heads=8, mem_dim=64, mem_vdim=128, groups=2, keep=1, decay_rank=32),
    "w2048": dict(kv_heads=8, window=1024, keep_first=4, streams=3, mem_heads=16, mem_dim=64, mem_vdim=128, groups=2, keep=1, decay_rank=32),
}


def vozetar_config(z, x):
    rot = {"base": 10000.0, "dims": z["dim"]}
    att = {"heads": z["heads"], "kv_heads": x["kv_heads"], "dim": z["dim"], "vdim": z["dim"], "scale": z["dim"] ** -0.5, "rot": rot}
    mask = {"size": x["window"], "keep_first": x["keep_first"]}
    ret = {"heads": x["mem_heads"], "dim": x["mem_dim"], "vdim": x["mem_vdim"], "rot": {"base": 10000.0, "dims": x["mem_dim"]},
           "decay": [1.0 - 2.0 ** (-5 - 5.0 * i / max(1, x["mem_heads"] - 1)) for i in range(x["mem_heads"])]}
    gla = {"heads": x["mem_heads"], "dim": x["mem_dim"], "vdim": x["mem_vdim"], "tau": 16.0, "decay_rank": x["decay_rank"]}
    par = {"left": dict(att, mask=mask), "left_scale": 1.0, "right": ret, "right_scale": 1.0}
    par2 = {"left": dict(att, mask=mask, conv=4), "right": gla}
    moe = {"kind": "moe", "expert": {"ff": z["expert_ff"]}, "shared": {"ff": z["shared_ff"]},
           "router": {"experts": z["experts"], "top": z["top"], "groups": {"count": x["groups"], "keep": x["keep"]}}}
    dense = {"kind": "dense", "ff": z["ff"]}
    return {"architecture": "Vozetar", "vocab": z["vocab"], "width": z["width"], "streams": x["streams"], "norm": {"eps": 1e-6},
            "embedding": {"bigram": {"buckets": 100003, "mul_prev": 8191, "mul_cur": 31}},
            "layers": [{"type": "attention", "mixer": dict(att, conv=3), "mlp": dense}, {"type": "parallel", "mixer": par, "mlp": moe},
                       {"type": "parallel_2", "mixer": par2, "mlp": dense}, {"type": "parallel", "mixer": par, "mlp": moe}]}


# ------------------------------------------------------------------------------------------------ --design zabozen
# The same widths, four layers with a norm on both sides of every sublayer and a SiLU-gated unit each: windowed attention with slopes by
# distance; latent attention with a rotated key part of 32 values and every earlier token visible; the gated delta rule; attention on the
# first layer's keys with a wider window.  Beside it Fidizen (the same latent attention kernels behind a query latent, with a window, a sink
# and routed experts), Vozetar (windowed attention and linear attention with a matrix memory side by side) and the Llama decoder at equal
# width and depth.
ZABOZEN_EXTRA = {
    "w1024": dict(kv_heads=4, window=1024, reader_window=1536, rot_dim=32, delta_heads=8, delta_kv_heads=4, delta_dim=128, delta_vdim=128, conv=4),
    "w2048": dict(kv_heads=8, window=1024, reader_window=1536, rot_dim=32, delta_heads=16, delta_kv_heads=8, delta_dim=128, delta_vdim=128, conv=4),
}


def zabozen_config(z, x):
    att = {"heads": z["heads"], "kv_heads": x["kv_heads"], "dim": z["dim"], "vdim": z["dim"], "scale": z["dim"] ** -0.5}
    lat = {"heads": z["heads"], "dim": z["dim"], "rot_dim": x["rot_dim"], "vdim": z["dim"], "kv_rank": z["kv_rank"],
           "scale": (z["dim"] + x["rot_dim"]) ** -0.5, "rot": {"base": 10000.0, "dims": x["rot_dim"]}}
    dlt = {"heads": x["delta_heads"], "kv_heads": x["delta_kv_heads"], "dim": x["delta_dim"], "vdim": x["delta_vdim"], "conv": x["conv"]}
    dense = {"kind": "dense", "ff": z["ff"]}
    return {"architecture": "Zabozen", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6}, "residual_mult": 0.8, "logit_softcap": 25.0,
            "layers": [{"type": "attention", "mixer": dict(att, mask={"size": x["window"]}), "mlp": dense},
                       {"type": "latent_attention", "mixer": lat, "mlp": dense}, {"type": "delta", "mixer": dlt, "mlp": dense},
                       {"type": "attention", "mixer": dict(att, mask={"size": x["reader_window"]}, kv_from=0), "mlp": dense}]}


# ------------------------------------------------------------------------------------------------ --design depunex
# The same widths, four layers with one norm for both sublayers and an input of the token's own: Mamba-2 + clamped gated unit; chunked
# attention beside the selective scan + routed experts; Mamba-2 + routed experts; the second layer's mixer + clamped gated unit.  Beside it
# Semesun (the same Mamba-2 sizes, windowed attention with the same kernels, routed experts in groups), Vozetar (two mixers side by side,
# the same pair table) and the Llama decoder at equal width and depth.
DEPUNEX_EXTRA = {
    "w1024": dict(kv_heads=4, chunk=1024, ssm_heads=32, ssm_vdim=64, ssm_state=128, ssm_groups=1, inner=2048, dt_rank=64, scan_state=16, token_dim=128,
                  groups=2, keep=1),
    "w2048": dict(kv_heads=8, chunk=1024, ssm_heads=64, ssm_vdim=64, ssm_state=128, ssm_groups=1, inner=4096, dt_rank=128, scan_state=16, token_dim=256,
                  groups=2, keep=1),
}


def depunex_config(z, x):
    att = {"heads": z["heads"], "kv_heads": x["kv_heads"], "dim": z["dim"], "vdim": z["dim"], "scale": z["dim"] ** -0.5, "mask": {"size": x["chunk"]},
           "rot": {"base": 500000.0, "dims": z["dim"], "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}
    scan = {"inner": x["inner"], "dt_rank": x["dt_rank"], "state": x["scan_state"], "conv": 4}
    par = {"left": att, "left_scale": 0.7, "right": scan, "right_scale": 0.7}
    ssm = {"heads": x["ssm_heads"], "vdim": x["ssm_vdim"], "state": x["ssm_state"], "groups": x["ssm_groups"], "conv": 4, "norm_groups": 1}
    moe = {"kind": "moe", "expert": {"ff": z["expert_ff"]},
           "router": {"experts": z["experts"], "top": z["top"], "groups": {"count": x["groups"], "keep": x["keep"]}}}
    dense = {"kind": "dense", "ff": z["ff"], "limit": 7.0}
    return {"architecture": "Depunex", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6}, "logit_softcap": 30.0, "token_side": {"dim": x["token_dim"]},
            "embedding": {"scale": z["width"] ** 0.5, "bigram": {"buckets": 100003, "mul_prev": 8191, "mul_cur": 31}},
            "layers": [{"type": "mamba2", "mixer": ssm, "mlp": dense}, {"type": "parallel", "mixer": par, "mlp": moe},
                       {"type": "mamba2", "mixer": ssm, "mlp": moe}, {"type": "parallel", "mixer": par, "mlp": dense}]}


def kogilix_attention_config(z):
    att = {"heads": z["heads"], "dim": z["dim"], "vdim": z["dim"], "q_rank": z["q_rank"], "kv_rank": z["kv_rank"], "scale": z["dim"] ** -0.5}
    moe = {"kind": "moe", "expert": {"ff": z["expert_ff"]}, "router": {"experts": z["experts"], "top": z["top"]}, "shared": {"ff": z["shared_ff"]}}
    dense = {"kind": "dense", "ff": z["ff"]}
    return {"architecture": "Kogilix", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6},
            "layers": [{"type": "latent_attention", "mixer": att, "mlp": mlp} for mlp in (dense, moe, dense, moe)]}


def llama_config_like(z):
    return {"architectures": ["LlamaForCausalLM"], "model_type": "llama", "num_hidden_layers": 4, "hidden_size": z["width"],
            "num_attention_heads": z["heads"], "num_key_value_heads": z["heads"], "intermediate_size": z["ff"], "vocab_size": z["vocab"],
            "rope_theta": 10000.0, "rms_norm_eps": 1e-6, "tie_word_embeddings": False, "max_position_embeddings": 8192}


def op_table(vm, engine, entries):
    """Device time per kind of operation of ONE step (two events around every launch): {name: [launches, ms]}."""
    with vm.OpTimes() as t:
        engine.step(entries)
        text = t.table()
    out = {}
    for line in text.splitlines()[1:]:
        cells = line.split()
        if len(cells) >= 3 and cells[0] != "total":
            out[cells[0]] = [int(cells[1]), float(cells[2])]
    return out


def design_arm(args):
    """Prompt and decode throughput of a design (Kogilix, Semesun, Fidizen, Vozetar, Zabozen, Depunex) at a few sizes, beside the library's other models at equal size."""
    import numpy as np
    import velomind_b200 as vm
    T, B, prompt_len = 2048, 8, 512
    steps, warmup = args.steps, max(args.warmup, 3)
    sizes = {}
    clock = ClockSampler()
    clock.start()
    for name, z in KOGILIX_SIZES.items():
        row = {}
        models = [("kogilix", kogilix_config(z)), ("llama", llama_config_like(z))]
        if args.design == "semesun":
            models.insert(0, ("semesun", semesun_config(z, SEMESUN_EXTRA[name])))
        if args.design == "vozetar":
            models = [("vozetar", vozetar_config(z, VOZETAR_EXTRA[name])), ("semesun", semesun_config(z, SEMESUN_EXTRA[name])), ("llama", llama_config_like(z))]
        if args.design == "zabozen":
            models = [("zabozen", zabozen_config(z, ZABOZEN_EXTRA[name])), ("fidizen", fidizen_config(z, FIDIZEN_EXTRA[name])),
                      ("vozetar", vozetar_config(z, VOZETAR_EXTRA[name])), ("llama", llama_config_like(z))]
        if args.design == "depunex":
            models = [("depunex", depunex_config(z, DEPUNEX_EXTRA[name])), ("semesun", semesun_config(z, SEMESUN_EXTRA[name])),
                      ("vozetar", vozetar_config(z, VOZETAR_EXTRA[name])), ("llama", llama_config_like(z))]
        if args.design == "fidizen":
            models = [("fidizen", fidizen_config(z, FIDIZEN_EXTRA[name])), ("kogilix_attention", kogilix_attention_config(z)), ("llama", llama_config_like(z))]
        for which, cfg in models:
            with tempfile.TemporaryDirectory(prefix="velomind_bench_") as folder:
                vm.write_random_model(folder, cfg, seed=0, std=0.02)
                te = vm.TextEngine(vm.EngineConfig(model_path=folder, dtype="bfloat16", max_tokens=B * 1024 + 4 * T, max_batch=B)).load()
            fresh = vm.Engine(te.model, T + 64, use_graphs=False)
            pms = prefill_run(fresh, T, z["vocab"])
            rng = np.random.default_rng(3)
            slot = fresh.open()
            prompt_ops = op_table(vm, fresh, [vm.Entry(slot, rng.integers(0, z["vocab"], T).tolist(), [T - 1])])
            fresh.close(slot)
            del fresh
            ms, _, launches, calls, _ = decode_run(te, B, prompt_len, steps, warmup, z["vocab"])
            eng = te.engine
            slots = [eng.open() for _ in range(B)]
            eng.step([vm.Entry(sl, rng.integers(0, z["vocab"], prompt_len).tolist(), []) for sl in slots])
            decode_ops = op_table(vm, eng, [vm.Entry(sl, [1], [0]) for sl in slots])
            for sl in slots:
                eng.close(sl)
            row[which] = {"prefill_tokens_per_s": T * 1000.0 / pms, "prefill_ms": pms, "decode_tokens_per_s": B * 1000.0 / ms, "decode_ms_per_step": ms,
                          "decode_launches_per_step": launches / steps, "decode_library_calls_per_step": calls / steps,
                          "prefill_ops": prompt_ops, "decode_ops": decode_ops}
            del te
        sizes[name] = dict(row, config=z)
    clocks = clock.stop()
    return {"design": args.design, "metric": "prompt tok/s (one prompt of 2,048 tokens, first-seen shape) and decode tok/s (batch 8, 512 cached tokens)",
            "unit": "tokens/s", "n_gpus": 1, "steps": steps, "warmup": warmup, "dtype": "bf16", "data": "synthetic", "layers": 4, "sizes": sizes,
            "clocks": clocks, "peaks": peaks()}


def _parse_reference_table(markdown: str):
    """Rows of the reference tool's report: {S: (prefill ms, prefill tok/s, decode ms, decode tok/s)} of the CUDA backend."""
    rows = {}
    for line in markdown.splitlines():
        cells = [c.strip() for c in line.strip().strip("|").split("|")]
        if len(cells) < 8 or cells[0] != "CUDA":
            continue
        try:
            S = int(cells[1])
            prefill_ms = float(cells[4].split("/")[0])
            prefill_tps = float(cells[5].split()[0])
            decode_ms = float(cells[6].split("/")[0])
            decode_tps = float(cells[7].split()[0])
        except (ValueError, IndexError):
            continue
        rows[S] = (prefill_ms, prefill_tps, decode_ms, decode_tps)
    return rows


def reference_arm(args):
    """The reference's own numbers for the same metric and sizes, or the one-line reason why there are none."""
    if args.gpus != 1:
        return {"impl": "reference", "unavailable": "the reference runs on one device only"}
    ref_dir = os.path.join(ROOT, "baseline", "_ref")
    tool, driver = os.path.join(ref_dir, "benchmark_baseline"), os.path.join(ref_dir, "reference_driver")
    if not (os.path.isfile(tool) and os.path.isfile(driver)):
        try:
            sys.path.insert(0, os.path.join(ROOT, "baseline"))
            import build_reference
            build_reference.build()
        except Exception as ex:      # no checkout of the reference, or no compiler
            return {"impl": "reference", "unavailable": f"the reference could not be built here: {str(ex).splitlines()[0][:200]}"}
    B, prompt_len, T = 8, 512, 2048
    steps, warmup = max(1, args.steps), max(args.warmup, 3)
    clock = ClockSampler()
    with tempfile.TemporaryDirectory(prefix="velomind_ref_") as work:
        report = os.path.join(work, "report.md")
        clock.start()
        # its own tool: median over `steps` executes after `warmup`; S = 512 gives decode at context 512, S = 2048 the prompt
        r = subprocess.run([tool, "--device", "cuda", "--synthetic", "--seq-lens", f"{prompt_len},{T}", "--iters", str(min(steps, 20)),
                            "--warmup", str(warmup), "--quiet", "--markdown", report], cwd=work, capture_output=True, text=True, timeout=1500)
        clocks = clock.stop()
        if r.returncode != 0 or not os.path.isfile(report):
            return {"impl": "reference", "unavailable": f"the reference's benchmark tool failed (exit {r.returncode}): {(r.stderr or r.stdout).strip().splitlines()[-1][:200] if (r.stderr or r.stdout).strip() else ''}"}
        with open(report) as f:
            rows = _parse_reference_table(f.read())
        if prompt_len not in rows or T not in rows:
            return {"impl": "reference", "unavailable": "the reference's report has no CUDA rows (no CUDA device?)"}
        # end to end through its public engine API: B sequences one after another, host tokens in, host logits out
        d = subprocess.run([driver, "cuda", str(B), str(prompt_len), str(min(steps, 20)), "3", str(T)], cwd=work, capture_output=True,
                           text=True, timeout=1500)
        e2e = None
        if d.returncode == 0:
            try:
                rec = json.loads(d.stdout.strip().splitlines()[-1])
                n = rec["sequences"] * rec["decode_steps"]
                e2e = {"value": n * 1000.0 / rec["decode_ms_total"], "unit": "tokens/s", "h2d_bytes_per_step": 4,
                       "d2h_bytes_per_step": rec["logit_bytes_per_step"], "ms_per_token": rec["decode_ms_median"],
                       "prefill_2048_ms": rec["prefill_ms_median"]}
            except (ValueError, KeyError, IndexError):
                e2e = None
    _, _, decode_ms, decode_tps = rows[prompt_len]
    prefill_ms, prefill_tps, _, _ = rows[T]
    pk = peaks()
    cfg = {"hidden_size": 576, "intermediate_size": 1536, "vocab_size": 49152, "num_attention_heads": 9, "num_key_value_heads": 3}
    per_layer, _, _, D = model_bytes_and_flops(cfg, 30)
    flops = 2.0 * T * per_layer * 30 + 4.0 * D * 9 * (T * (T + 1) / 2.0) * 30 + 2.0 * 49152 * 576
    line = {
        "impl": "reference",
        "metric": "decode tok/s at batch 8 (SmolLM2-135M shape, prompts of 512 tokens)",
        "value": decode_tps, "unit": "tokens/s", "n_gpus": 1, "steps": min(steps, 20), "warmup": warmup,
        "ms_per_step": decode_ms * B, "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "fp32",
        "data": "synthetic",
        "config": {"model": "SmolLM2-135M shape, the reference's own --synthetic weights", "global_batch": B, "seq_len": prompt_len,
                   "parallelism": "single GPU", "layers": 30, "layers_of_config": 30, "hidden": 576, "heads": 9, "kv_heads": 3,
                   "head_dim": 64, "intermediate": 1536, "vocab": 49152,
                   "batching": "none in the reference: 8 sequences one after another, tokens/s equal its batch-1 figure",
                   "timing": "the reference's own tool: host clock around one execute of its decode graph, median",
                   "built_from": "unmodified sources, CUDA backend for sm_100, cuBLAS float32"},
        "prefill": {"value": prefill_tps, "tokens": T, "ms": prefill_ms, "frac": flops / (prefill_ms * 1e-3) / (pk["bf16_tflops"] * 1e12)},
        "points": {"decode_b1": decode_tps, "decode_b64": decode_tps},
        "clocks": clocks,
        "gpu_launches": 0,
    }
    if e2e is not None:
        line["e2e"] = e2e
    return line


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--layers", type=int, default=0, help="fewer layers than the configuration (0: all); reported in config")
    ap.add_argument("--quick", action="store_true", help="skip the batch 1 / 64 points and the end-to-end run")
    ap.add_argument("--shape", default="135m", choices=sorted(SHAPES),
                    help="sizes of the random model: the benchmark's SmolLM2-135M (default), or the 360M / 1.7B shapes of the family")
    ap.add_argument("--design", default="", choices=["", "kogilix", "semesun", "fidizen", "vozetar", "zabozen", "depunex"],
                    help="instead of the benchmark: prompt and decode throughput of another design of the library at a few layer sizes, "
                         "beside the Llama decoder at equal size (one JSON line of its own)")
    args = ap.parse_args()

    if args.design:
        if args.gpus != 1:
            print(f"bench.py measures a single-GPU library: --gpus {args.gpus} is not supported, run with --gpus 1")
            return 2
        print(json.dumps(design_arm(args)))
        return 0
    if args.impl == "reference":
        print(json.dumps(reference_arm(args)))
        return 0
    if args.gpus != 1:
        print(f"bench.py measures a single-GPU library: --gpus {args.gpus} is not supported, run with --gpus 1")
        return 2
    warmup = max(args.warmup, 3)

    import numpy as np
    import velomind_b200 as vm

    cfg = dict(vm.SMOLLM2_135M)
    cfg.update(SHAPES[args.shape])
    full_layers = cfg["num_hidden_layers"]
    layers = args.layers or full_layers
    cfg["num_hidden_layers"] = layers
    vocab = cfg["vocab_size"]
    B, prompt_len, context = 8, 512, 4096
    pk = peaks()

    with tempfile.TemporaryDirectory(prefix="velomind_bench_") as folder:
        vm.write_random_model(folder, cfg, seed=0, std=0.02)
        te = vm.TextEngine(vm.EngineConfig(model_path=folder, dtype="bfloat16", max_tokens=64 * context + 8192, max_batch=64)).load()

    per_layer, weight_bytes, kv_per_token, D = model_bytes_and_flops(cfg, layers)

    clock = ClockSampler()
    ms, mean_ctx, launches, calls, clocks = decode_run(te, B, prompt_len, args.steps, warmup, vocab, clock)
    value = B * 1000.0 / ms
    step_bytes = weight_bytes + kv_per_token * mean_ctx * B
    achieved = step_bytes / (ms * 1e-3) / 1e9

    # prefill of 2,048 tokens: linears + causal attention + the head on one row.  The headline figure is a FIRST-SEEN shape: the
    # step's kernels launched one by one from the host, which is what a prompt of a new length gets; the same step replayed from
    # its CUDA graph (what a repeated shape gets) goes to `points`.
    T = 2048
    fresh = vm.Engine(te.model, T + 64, use_graphs=False)
    pms = prefill_run(fresh, T, vocab)
    del fresh
    H = cfg["num_attention_heads"]
    flops = 2.0 * T * per_layer * layers + 4.0 * D * H * (T * (T + 1) / 2.0) * layers + 2.0 * vocab * cfg["hidden_size"]
    prefill = {"value": T * 1000.0 / pms, "tokens": T, "ms": pms, "frac": flops / (pms * 1e-3) / (pk["bf16_tflops"] * 1e12)}

    points, e2e = {}, None
    if not args.quick:
        replayed_ms = prefill_run(te.engine, T, vocab)
        points["prefill_2048_replayed"] = T * 1000.0 / replayed_ms
        for b in (1, 64):
            m, _, _, _, _ = decode_run(te, b, prompt_len, args.steps, warmup, vocab)
            points[f"decode_b{b}"] = b * 1000.0 / m
        # end to end through the public entry point: host token ids in, host token ids out
        rng = np.random.default_rng(1)
        prompts = [rng.integers(0, vocab, prompt_len).tolist() for _ in range(B)]
        # the host reads every step's tokens and sends the next step's descriptors (steps_per_sync=1): an end-to-end step includes both
        te.generate(prompts, temperature=0.0, max_tokens=warmup + 1, stop_tokens=(), steps_per_sync=1)
        # bytes are counted where they are copied (descriptors and sampler parameters up, sampled tokens down); what the
        # prompt step alone moves is taken off, as the timed region is the decode steps
        c0 = te.engine.counters
        te.generate(prompts, temperature=0.0, max_tokens=1, stop_tokens=(), steps_per_sync=1)
        c1 = te.engine.counters
        h2d_prompt, d2h_prompt = c1["h2d_bytes"] - c0["h2d_bytes"], c1["d2h_bytes"] - c0["d2h_bytes"]
        te.generate(prompts, temperature=0.0, max_tokens=args.steps + 1, stop_tokens=(), steps_per_sync=1)
        c2 = te.engine.counters
        tm = te.last_timing
        e2e = {"value": B * tm.decode_steps / tm.decode_seconds, "unit": "tokens/s",
               "h2d_bytes_per_step": round((c2["h2d_bytes"] - c1["h2d_bytes"] - h2d_prompt) / max(tm.decode_steps, 1)),
               "d2h_bytes_per_step": round((c2["d2h_bytes"] - c1["d2h_bytes"] - d2h_prompt) / max(tm.decode_steps, 1))}
        # the same call with 8 decode steps queued per host round trip
        te.generate(prompts, temperature=0.0, max_tokens=args.steps + 1, stop_tokens=(), steps_per_sync=8)
        points["e2e_queued_8"] = B * te.last_timing.decode_steps / te.last_timing.decode_seconds
        if args.shape == "360m":
            # BASELINE.json's run at this shape: batch 16, prompt lengths uniform in [64, 1024], 256 decode steps
            dec, pre, n_prompt = unequal_batch_run(te, 16, 64, 1024, 256, vocab)
            points["unequal_b16_decode"] = dec
            points["unequal_b16_prompt_tokens_per_s"] = pre
        if args.shape == "1.7b":
            # BASELINE.json's run at this shape: decode at batch 1 / 8 / 64 up to context 4096
            for b in (1, 8, 64):
                m, _, _, _, _ = decode_run(te, b, prompt_len, min(args.steps, 32), 3, vocab, context_fill=context - 64)
                points[f"decode_b{b}_ctx4096"] = b * 1000.0 / m
    line = {
        "metric": f"decode tok/s at batch 8 (SmolLM2-{args.shape.upper()} shape, prompts of 512 tokens)",
        "value": value, "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": warmup, "ms_per_step": ms,
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
        "config": {"model": f"SmolLM2-{args.shape.upper()} shape, random weights", "global_batch": B, "seq_len": prompt_len, "context": context,
                   "parallelism": "single GPU", "layers": layers, "layers_of_config": full_layers,
                   "hidden": cfg["hidden_size"], "heads": H, "kv_heads": cfg["num_key_value_heads"], "head_dim": D,
                   "intermediate": cfg["intermediate_size"], "vocab": vocab, "rope_theta": cfg["rope_theta"],
                   "rms_eps": cfg["rms_norm_eps"], "tied_embeddings": True, "sampling": "greedy on device",
                   "prefill_shape": "first seen (kernels launched one by one); points.prefill_2048_replayed: from its CUDA graph",
                   "l2": "inputs larger than L2 (weights + cache > 126 MB)", "peaks": pk["source"]},
        "prefill": prefill,
        "roofline": {"bound": "hbm", "achieved": achieved, "peak": pk["hbm_gbs"], "unit": "GB/s", "frac": achieved / pk["hbm_gbs"]},
        "points": points,
        "clocks": clocks,
        "gpu_launches": launches,
        "library_gemm_calls": calls,
    }
    if e2e is not None:
        line["e2e"] = e2e
    print(json.dumps(line))
    return 0


if __name__ == "__main__":
    sys.exit(main())
