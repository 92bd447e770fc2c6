#!/usr/bin/env python3
"""Headline measurement: LFM2-1.2B layer sizes, random bfloat16 weights, one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference]

A "step" is one decode step of a batch of 8 requests, each with a 2,048-token prompt in
the cache (context length 4,096, pages of 16 tokens).  `value` is decoded tokens per
second over exactly K steps, timed on the device with CUDA events after W warm-up steps;
the step's inputs are larger than L2 (2.3 GB of weights are read every step), so no
flush is needed between iterations.  `e2e` is the same metric through Engine.generate:
host token lists in, host token lists out, with the per-step host-to-device copy of the
batch descriptor and device-to-host copy of the sampled ids inside the timed region.
One JSON line is printed.  For --gpus N > 1 one line says that this engine is a
one-GPU engine and the exit code is 2.

`prefill` times one 2,048-token prompt per repetition (a new request each time, CUDA events
around the step); from its third run on the step is replayed from the graph the engine
captured for its shape, as every step whose shape repeats is.

--workload continuous | long run the baseline's two other workloads (LFM2-700M sizes under
continuous batching; LFM2-350M sizes with 32,768-token prompts in bfloat16 and 32-bit) and
print one JSON line each; --workload sizes runs the headline's model at further prompt lengths
and decode contexts; --workload vipotar / negotar run the Vipotar / Negotar design at two sizes that resemble a real model's layers beside
LFM2 at equal width, depth, heads and feed-forward size (prefill of one prompt, decode at batch 8), --workload keralix the
Keralix design beside Vipotar likewise, --workload zepesun the Zepesun design beside Negotar, --workload modinex the Modinex design beside Vipotar,
--workload zinunex the Zinunex design beside Zepesun (--only-size NAME: one of its sizes); the default is the headline above.
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

# the config.json of LFM2-1.2B (the sizes the headline is quoted on); weights are random
with open(os.path.join(ROOT, "imparo_b200", "config", "presets", "lfm2_1.2b.json")) as _f:
    LFM2_1_2B = json.load(_f)
PROMPT = 2048
CTX = 4096
PAGE = 16
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    try:
        with open(path) as f:
            d = json.load(f)
        return {"hbm_gbs": float(d["hbm_gbs"]), "bf16_tflops": float(d.get("bf16_tflops_sustained") or d["bf16_tflops"]),
                "bf16_tflops_burst": float(d["bf16_tflops"]), "source": "measured"}
    except Exception:
        return dict(FALLBACK_PEAKS, bf16_tflops_burst=FALLBACK_PEAKS["bf16_tflops"], source="fallback")


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while a region is timed."""
    FIELDS = ("clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
              "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, index=0):
        self.rows, self.proc, self.index = [], None, index

    def __enter__(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", f"--query-gpu={self.FIELDS}", "--format=csv,noheader,nounits",
                                          "-i", str(self.index), "-lms", "100"], stdout=subprocess.PIPE,
                                         stderr=subprocess.DEVNULL, text=True)
            self.thread = threading.Thread(target=self._read, daemon=True)
            self.thread.start()
        except OSError:
            self.proc = None
        return self

    def _read(self):
        for line in self.proc.stdout:
            parts = [p.strip() for p in line.split(",")]
            if len(parts) >= 7:
                self.rows.append(parts)

    def __exit__(self, *a):
        if self.proc is not None:
            time.sleep(0.15)
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()

    def summary(self):
        sm, mx, reasons = [], [], set()
        for r in self.rows:
            try:
                sm.append(float(r[0])); mx.append(float(r[1]))
            except ValueError:
                continue
            for name, v in zip(("hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"), r[3:7]):
                if v.lower().startswith("active"):
                    reasons.add(name)
        if not sm:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["unsampled"]}
        return {"sm_mhz": statistics.median(sm), "sm_max_mhz": max(mx), "reasons": sorted(reasons), "samples": len(sm)}


def model_numbers(engine):
    """Bytes a decode step must read for its weights, KV bytes per cached token, and the
    flops of a prompt of T tokens, from the model's own parts."""
    cfg = engine.config
    H, F, V = cfg.hidden_size, cfg.ff_dim, cfg.vocab_size
    nh, nkv, hd = cfg.num_attention_heads, cfg.num_key_value_heads, cfg.head_dim
    n_attn = sum(1 for e in engine.model.schedule if cfg.layer_types[e.layer] != "conv")
    n_conv = len(engine.model.schedule) - n_attn
    per_layer_ffn = 3 * H * F
    conv = 3 * H * H + H * H
    attn = (nh + 2 * nkv) * hd * H + H * nh * hd
    matrix_params = len(engine.model.schedule) * per_layer_ffn + n_conv * conv + n_attn * attn
    elt = 2 if engine.precision == "bfloat16" else 4
    weight_bytes = (matrix_params + V * H) * elt          # every matrix once; the tied table is the head
    kv_per_token = n_attn * 2 * nkv * hd * elt

    def prefill_flops(T, wanted=1):
        # what the step executes: the last layer's feed-forward runs on the wanted rows only (as
        # in the reference), every other product on all T tokens; causal attention; the head on the wanted rows
        return 2.0 * T * (matrix_params - per_layer_ffn) + 2.0 * wanted * per_layer_ffn + 2.0 * wanted * V * H \
            + n_attn * 4.0 * nh * hd * T * (T + 1) / 2
    return weight_bytes, kv_per_token, prefill_flops, matrix_params + V * H


def measure_decode(engine, batch, steps, warmup, rng, sampler=None, prompt=None):
    """-> (ms per step, launches per step, h2d bytes per step, mean context) with `batch`
    requests holding `prompt` (default PROMPT) tokens each."""
    PROMPT = prompt or globals()["PROMPT"]
    import torch
    from imparo_b200.engine import StepItem
    from imparo_b200.kernels import ops
    ids = list(range(1000 * batch, 1000 * batch + batch))
    V = engine.vocab_size
    for r in ids:
        engine.add_request(r)
        engine.step([StepItem(r, rng.integers(0, V, PROMPT).tolist(), [PROMPT - 1])])
    out_ids = torch.empty(batch, dtype=torch.int32, device=engine.device)

    def one():
        logits = engine.step_fn([StepItem(r, [int(t)], [0]) for r, t in zip(ids, rng.integers(0, V, batch))])
        ops.sample_rows(logits, None, None, out_ids)
    for _ in range(max(warmup, 3)):
        one()
    torch.cuda.synchronize()
    before = dict(ops.COUNTS)
    start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    start.record()
    for _ in range(steps):
        one()
    end.record()
    torch.cuda.synchronize()
    ms = start.elapsed_time(end) / steps
    launches = (ops.COUNTS["own"] - before["own"]) / steps
    library = (ops.COUNTS["library"] - before["library"]) / steps
    ctx = PROMPT + max(warmup, 3) + steps / 2.0
    engine.check_device_status()
    for r in ids:
        engine.end_request(r)
    return ms, launches, library, ctx


def measure_prefill(engine, reps, warmup, rng, prompt=None):
    import torch
    PROMPT = prompt or globals()["PROMPT"]
    from imparo_b200.engine import StepItem
    V = engine.vocab_size
    times = []
    for i in range(warmup + reps):
        toks = rng.integers(0, V, PROMPT).tolist()
        engine.add_request(77000 + i)
        torch.cuda.synchronize()
        start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        start.record()
        engine.step_fn([StepItem(77000 + i, toks, [PROMPT - 1])])
        end.record()
        torch.cuda.synchronize()
        engine.end_request(77000 + i)
        if i >= warmup:
            times.append(start.elapsed_time(end))
    return statistics.median(times)


def measure_e2e(engine, batch, steps, warmup, rng):
    """Decode tokens per second through Engine.generate: wall clock from the end of decode
    step `warmup` to the end of decode step `warmup + steps`, host lists in and out."""
    V = engine.vocab_size
    prompts = [rng.integers(0, V, PROMPT).tolist() for _ in range(batch)]
    stamps, h2d = [], []

    def on_step(plan):
        if all(e.count == 1 for e in plan) and len(plan) == batch:
            stamps.append(time.perf_counter())
            h2d.append(engine.step_fn.last_h2d_bytes)       # this step's batch description, as uploaded
    n_new = warmup + steps + 2 + 2 * batch      # requests start decoding up to ~batch steps apart
    out = engine.generate(prompts, max_tokens=n_new, on_step=on_step, stop_token_ids=[])
    assert all(len(o) == n_new for o in out) and len(stamps) > warmup + steps, (len(stamps), warmup + steps)
    dt = stamps[warmup + steps] - stamps[warmup]
    return batch * steps / dt, max(h2d[warmup:warmup + steps + 1])


def workload_sizes(args):
    """LFM2-1.2B layer sizes (all 16 layers, random bfloat16 weights) at further sizes than the headline: one prompt
    of 512, 2,048, 8,192 and 32,768 tokens (tokens per second; flops over time against the measured bfloat16 peak), and
    decode steps of 8 requests at contexts of 2,048, 16,384 and 32,768 tokens (tokens per second; bytes the step has
    to read over its time against the measured HBM peak)."""
    import numpy as np
    import torch
    from imparo_b200.engine import Engine
    rng = np.random.default_rng(0)
    pk = peaks()
    longest = 32768
    engine = Engine(config=dict(LFM2_1_2B), seed=0, dtype="bfloat16", ctx=longest + 256, parallel=8, page_size=PAGE,
                    max_step_tokens=longest, random_init={"norm_jitter": 0.0})
    weight_bytes, kv_per_token, prefill_flops, n_params = model_numbers(engine)
    out = {"metric": "LFM2-1.2B at further sizes: prefill of one prompt, decode at batch 8", "unit": "tokens/s", "dtype": "bf16",
           "data": "synthetic (random weights, uniform-random token ids)", "prefill": {}, "decode_b8": {}}
    with ClockSampler() as clocks:
        for T in (512, 2048, 8192, 32768):
            ms = measure_prefill(engine, reps=3 if T > 8192 else 5, warmup=3, rng=rng, prompt=T)
            out["prefill"][str(T)] = {"value": round(T * 1000.0 / ms, 1), "ms": round(ms, 3),
                                      "frac": round(prefill_flops(T) / (ms * 1e-3) / (pk["bf16_tflops_burst"] * 1e12), 4)}
        for ctx_len in (2048, 16384, 32768):
            ms, _, _, ctx = measure_decode(engine, 8, 30, 5, rng, prompt=ctx_len)
            nbytes = weight_bytes + 8 * ctx * kv_per_token
            out["decode_b8"][str(ctx_len)] = {"value": round(8 * 1000.0 / ms, 1), "ms_per_step": round(ms, 4),
                                              "roofline": {"bound": "hbm", "achieved": round(nbytes / (ms * 1e-3) / 1e9, 1),
                                                           "peak": pk["hbm_gbs"], "unit": "GB/s",
                                                           "frac": round(nbytes / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}}
    out["peaks"] = pk["source"]
    out["config"] = {"model": "LFM2-1.2B", "layers": 16, "layers_of_config": 16, "page_size": PAGE, "params": n_params}
    out["clocks"] = clocks.summary()
    print(json.dumps(out))
    return 0


def vipotar_config(width, layers, heads, kv_heads, head, window, lin_heads, lin_dim, lin_vdim, ff, vocab):
    """A Vipotar config.json of the given sizes: every layer the same, no repeated stretch, half of each head rotated
    with scaled frequencies, decays spread between 0.9 and 0.999."""
    left = {"heads": heads, "kv_heads": kv_heads, "dim": head, "vdim": head, "scale": head ** -0.5, "mask": {"size": window},
            "rot": {"dims": head // 2, "base": 500000.0, "scaling": {"factor": 4.0, "original": 2048, "fast": 32.0, "slow": 1.0}}}
    decay = [1.0 - 0.1 * (0.01 ** (h / max(lin_heads - 1, 1))) for h in range(lin_heads)]
    right = {"heads": lin_heads, "dim": lin_dim, "vdim": lin_vdim, "decay": decay}
    layer = {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": {"kind": "dense", "ff": ff}}
    return {"architecture": "Vipotar", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "residual_mult": 0.5,
            "logit_softcap": 30.0, "layers": [layer] * layers}


def lfm2_like(width, layers, heads, kv_heads, head, ff, vocab):
    """LFM2 at the same width, depth, heads and feed-forward size: two layers in three are short convolutions."""
    types = ["full_attention" if i % 3 == 2 else "conv" for i in range(layers)]
    return {"architectures": ["Lfm2ForCausalLM"], "model_type": "lfm2", "vocab_size": vocab, "hidden_size": width,
            "num_hidden_layers": layers, "layer_types": types, "num_attention_heads": heads, "num_key_value_heads": kv_heads,
            "head_dim": head, "block_ff_dim": ff, "block_auto_adjust_ff_dim": False, "conv_L_cache": 3, "conv_bias": False,
            "rope_theta": 1000000.0, "norm_eps": 1e-5, "tie_embedding": True, "max_position_embeddings": 128000}


def workload_vipotar(args):
    """Vipotar at two sizes beside LFM2 at equal sizes: prefill of one prompt of 512 and 2,048 tokens, decode steps of 8
    requests with 2,048 positions each.  Rooflines: prefill against the measured bfloat16 peak with the flops the design
    needs (products over all tokens, attention over the window, the linear attention's 4 * heads * dim * vdim per token);
    decode against the measured copy bandwidth with the bytes a step must move (every matrix once, the windows' keys and
    values, the linear attention's states read and written)."""
    import numpy as np
    import torch
    from imparo_b200.engine import Engine
    rng = np.random.default_rng(0)
    pk = peaks()
    sizes = {"width1024": dict(width=1024, layers=8, heads=16, kv_heads=4, head=64, window=512, lin_heads=8, lin_dim=64, lin_vdim=128,
                               ff=4096, vocab=32768),
             "width2048": dict(width=2048, layers=8, heads=32, kv_heads=8, head=64, window=1024, lin_heads=16, lin_dim=128, lin_vdim=128,
                               ff=8192, vocab=65536)}
    out = {"metric": "Vipotar beside LFM2 at equal sizes: prefill of one prompt, decode at batch 8 with 2,048 positions",
           "unit": "tokens/s", "dtype": "bf16", "data": "synthetic (random weights, uniform-random token ids)", "sizes": {}}
    with ClockSampler() as clocks:
        for name, z in sizes.items():
            row = {}
            W, L, F, V = z["width"], z["layers"], z["ff"], z["vocab"]
            for model in ("vipotar", "lfm2"):
                if model == "vipotar":
                    cfg = vipotar_config(**z)
                    qkv = (z["heads"] + 2 * z["kv_heads"]) * z["head"] * W + W * z["heads"] * z["head"]
                    lin = (2 * z["lin_heads"] * z["lin_dim"] + 2 * z["lin_heads"] * z["lin_vdim"]) * W + W * z["lin_heads"] * z["lin_vdim"]
                    matrix = L * (qkv + lin + 2 * W * F)
                    state = L * z["lin_heads"] * z["lin_dim"] * z["lin_vdim"] * 4
                    kv_tok = L * 2 * z["kv_heads"] * z["head"] * 2
                    head_params = V * W

                    def flops(T):
                        keys = sum(min(t + 1, z["window"]) for t in range(T))
                        return 2.0 * T * matrix + 2.0 * V * W + L * (4.0 * z["heads"] * z["head"] * keys
                                                                     + 4.0 * z["lin_heads"] * z["lin_dim"] * z["lin_vdim"] * T)

                    def step_bytes(batch, ctx):
                        return (matrix + head_params) * 2 + batch * (2 * state + min(ctx, z["window"]) * kv_tok)
                else:
                    cfg = lfm2_like(W, L, z["heads"], z["kv_heads"], z["head"], F, V)
                    n_attn = sum(1 for t in cfg["layer_types"] if t != "conv")
                    attn = (z["heads"] + 2 * z["kv_heads"]) * z["head"] * W + W * z["heads"] * z["head"]
                    matrix = L * 3 * W * F + (L - n_attn) * 4 * W * W + n_attn * attn
                    kv_tok = n_attn * 2 * z["kv_heads"] * z["head"] * 2

                    def flops(T):
                        return 2.0 * T * matrix + 2.0 * V * W + n_attn * 4.0 * z["heads"] * z["head"] * T * (T + 1) / 2

                    def step_bytes(batch, ctx):
                        return (matrix + V * W) * 2 + batch * ctx * kv_tok
                engine = Engine(config=cfg, seed=0, dtype="bfloat16", ctx=CTX, parallel=8, page_size=PAGE, max_step_tokens=PROMPT,
                                random_init={"norm_jitter": 0.0})
                r = {"params": matrix + V * W * (2 if model == "vipotar" else 1), "prefill": {}}
                for T in (512, 2048):
                    ms = measure_prefill(engine, reps=5, warmup=3, rng=rng, prompt=T)
                    r["prefill"][str(T)] = {"value": round(T * 1000.0 / ms, 1), "ms": round(ms, 3),
                                            "frac": round(flops(T) / (ms * 1e-3) / (pk["bf16_tflops_burst"] * 1e12), 4)}
                ms, launches, library, ctx = measure_decode(engine, 8, max(20, args.steps // 4), max(args.warmup, 3), rng, prompt=PROMPT)
                nbytes = step_bytes(8, ctx)
                r["decode_b8"] = {"value": round(8 * 1000.0 / ms, 1), "ms_per_step": round(ms, 4), "own_kernels_per_step": round(launches, 1),
                                  "library_gemms_per_step": round(library, 1), "bytes_per_step": int(nbytes),
                                  "frac": round(nbytes / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}
                row[model] = r
                del engine
                torch.cuda.empty_cache()
            out["sizes"][name] = dict(row, config=z)
    out["peaks"] = pk["source"]
    out["clocks"] = clocks.summary()
    print(json.dumps(out))
    return 0


def negotar_config(width, layers, heads, kv_heads, head, ssm_heads, ssm_vdim, ssm_state, experts, top, ff, vocab):
    """A Negotar config.json of the given sizes: attention and state-space layers in turn (the first an attention layer),
    every head rotated with rescaled frequencies, scores capped at 50, values shared from the first attention layer,
    `experts` experts of `ff` features of which a token uses `top`."""
    attn = {"heads": heads, "kv_heads": kv_heads, "dim": head, "vdim": head, "scale": head ** -0.5 * 8.0, "softcap": 50.0,
            "v_mix": True, "rot": {"dims": head, "base": 500000.0, "scaling": {"factor": 4.0, "low": 1.0, "high": 8.0, "original": 4096}}}
    ssm = {"heads": ssm_heads, "vdim": ssm_vdim, "state": ssm_state, "groups": 1, "conv": 4, "norm_groups": 1}
    mlp = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    return {"architecture": "Negotar", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "logit_scale": 1.0,
            "layers": [{"type": "attention" if i % 2 == 0 else "mamba2", "mixer": attn if i % 2 == 0 else ssm, "mlp": mlp}
                       for i in range(layers)]}


def workload_negotar(args):
    """Negotar at two sizes beside LFM2 at equal width, depth, heads and active feed-forward size (top * ff): prefill of one
    prompt of 512 and 2,048 tokens, decode steps of 8 requests with 2,048 positions each.  Rooflines: prefill against the
    measured bfloat16 peak with the flops the design needs (products over all tokens, experts over the tokens that use
    them, causal attention, the recurrence's 6 * heads * state * vdim per token); decode against the measured copy
    bandwidth with the bytes a step must move (every dense matrix once, the experts the step's rows can reach at most,
    the keys and values, the recurrent states read and written)."""
    import numpy as np
    import torch
    from imparo_b200.engine import Engine
    rng = np.random.default_rng(0)
    pk = peaks()
    sizes = {"width1024": dict(width=1024, layers=8, heads=16, kv_heads=4, head=64, ssm_heads=32, ssm_vdim=64, ssm_state=64,
                               experts=16, top=2, ff=1024, vocab=32768),
             "width2048": dict(width=2048, layers=8, heads=32, kv_heads=8, head=64, ssm_heads=64, ssm_vdim=64, ssm_state=128,
                               experts=32, top=4, ff=1024, vocab=65536)}
    out = {"metric": "Negotar beside LFM2 at equal sizes: prefill of one prompt, decode at batch 8 with 2,048 positions",
           "unit": "tokens/s", "dtype": "bf16", "data": "synthetic (random weights, uniform-random token ids)", "sizes": {}}
    with ClockSampler() as clocks:
        for name, z in sizes.items():
            row = {}
            W, L, V = z["width"], z["layers"], z["vocab"]
            F = z["top"] * z["ff"]
            for model in ("negotar", "lfm2"):
                if model == "negotar":
                    cfg = negotar_config(**z)
                    n_attn = (L + 1) // 2
                    n_ssm = L - n_attn
                    inner, N = z["ssm_heads"] * z["ssm_vdim"], z["ssm_state"]
                    attn = (z["heads"] + 2 * z["kv_heads"]) * z["head"] * W + W * z["heads"] * z["head"]
                    ssm = (2 * inner + 2 * N + z["ssm_heads"]) * W + W * inner
                    expert = 3 * W * z["ff"]
                    dense = n_attn * attn + n_ssm * ssm + L * z["experts"] * W
                    state = n_ssm * z["ssm_heads"] * N * z["ssm_vdim"] * 4
                    kv_tok = n_attn * 2 * z["kv_heads"] * z["head"] * 2
                    params = dense + L * z["experts"] * expert + V * W

                    def flops(T):
                        return (2.0 * T * (dense + L * z["top"] * expert) + 2.0 * V * W
                                + n_attn * 4.0 * z["heads"] * z["head"] * T * (T + 1) / 2 + n_ssm * 6.0 * inner * N * T)

                    def step_bytes(batch, ctx):
                        reached = min(z["experts"], batch * z["top"])
                        return (dense + L * reached * expert + V * W) * 2 + batch * (2 * state + ctx * kv_tok)
                else:
                    cfg = lfm2_like(W, L, z["heads"], z["kv_heads"], z["head"], F, V)
                    n_attn = sum(1 for t in cfg["layer_types"] if t != "conv")
                    attn = (z["heads"] + 2 * z["kv_heads"]) * z["head"] * W + W * z["heads"] * z["head"]
                    matrix = L * 3 * W * F + (L - n_attn) * 4 * W * W + n_attn * attn
                    kv_tok = n_attn * 2 * z["kv_heads"] * z["head"] * 2
                    params = matrix + V * W

                    def flops(T):
                        return 2.0 * T * matrix + 2.0 * V * W + n_attn * 4.0 * z["heads"] * z["head"] * T * (T + 1) / 2

                    def step_bytes(batch, ctx):
                        return (matrix + V * W) * 2 + batch * ctx * kv_tok
                engine = Engine(config=cfg, seed=0, dtype="bfloat16", ctx=CTX, parallel=8, page_size=PAGE, max_step_tokens=PROMPT,
                                random_init={"norm_jitter": 0.0})
                r = {"params": params, "prefill": {}}
                for T in (512, 2048):
                    ms = measure_prefill(engine, reps=5, warmup=3, rng=rng, prompt=T)
                    r["prefill"][str(T)] = {"value": round(T * 1000.0 / ms, 1), "ms": round(ms, 3),
                                            "frac": round(flops(T) / (ms * 1e-3) / (pk["bf16_tflops_burst"] * 1e12), 4)}
                ms, launches, library, ctx = measure_decode(engine, 8, max(20, args.steps // 4), max(args.warmup, 3), rng, prompt=PROMPT)
                nbytes = step_bytes(8, ctx)
                r["decode_b8"] = {"value": round(8 * 1000.0 / ms, 1), "ms_per_step": round(ms, 4), "own_kernels_per_step": round(launches, 1),
                                  "library_gemms_per_step": round(library, 1), "bytes_per_step": int(nbytes),
                                  "frac": round(nbytes / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}
                row[model] = r
                del engine
                torch.cuda.empty_cache()
            out["sizes"][name] = dict(row, config=z)
    out["peaks"] = pk["source"]
    out["clocks"] = clocks.summary()
    print(json.dumps(out))
    return 0


def keralix_config(width, layers, streams, heads, kv_heads, head, window, lat_heads, lat_dim, lat_vdim, q_rank, kv_rank,
                   delta_heads, delta_kv_heads, delta_dim, delta_vdim, inner, ff, vocab):
    """A Keralix config.json of the given sizes: layers in the order delta rule, windowed attention, latent attention, latent
    attention, each with a dense feed-forward; `streams` copies of the stream; half of each attention head rotated; scores
    capped at 50; four conv taps."""
    attn = {"heads": heads, "kv_heads": kv_heads, "dim": head, "vdim": head, "conv": 4, "scale": head ** -0.5, "softcap": 50.0,
            "mask": {"size": window}, "rot": {"dims": head // 2, "base": 1000000.0}}
    latent = {"heads": lat_heads, "dim": lat_dim, "vdim": lat_vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": lat_dim ** -0.5}
    delta = {"heads": delta_heads, "kv_heads": delta_kv_heads, "dim": delta_dim, "vdim": delta_vdim, "conv": 4,
             "decay_rank": inner, "gate_rank": inner}
    kinds = [("channel_delta", delta), ("attention", attn), ("latent_attention", latent), ("latent_attention", latent)]
    return {"architecture": "Keralix", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "streams": streams,
            "embedding": {"scale": float(width) ** 0.5},
            "layers": [{"type": kinds[i % 4][0], "mixer": kinds[i % 4][1], "mlp": {"kind": "dense", "ff": ff}} for i in range(layers)]}


def workload_keralix(args):
    """Keralix at two sizes beside Vipotar (windowed attention next to a recurrent linear attention, dense feed-forward: the
    closest design the engine serves) at equal width, depth, attention heads, window, recurrent state size and feed-forward
    size: prefill of one prompt of 512 and 2,048 tokens, decode steps of 8 requests with 2,048 positions each.  Rooflines:
    prefill against the measured bfloat16 peak with the flops the design needs (products over all tokens, attention over
    the window, the latent attention in its latent space over all earlier positions, the delta rule's 7 * heads * dim * vdim
    per token); decode against the measured copy bandwidth with the bytes a step must move (every matrix once, the windows'
    keys, the latents, the recurrent states read and written)."""
    import numpy as np
    import torch
    from imparo_b200.engine import Engine
    rng = np.random.default_rng(0)
    pk = peaks()
    sizes = {"width1024": dict(width=1024, layers=8, streams=4, heads=16, kv_heads=4, head=64, window=512, lat_heads=16, lat_dim=64,
                               lat_vdim=64, q_rank=384, kv_rank=128, delta_heads=8, delta_kv_heads=4, delta_dim=64, delta_vdim=128,
                               inner=64, ff=4096, vocab=32768),
             "width2048": dict(width=2048, layers=8, streams=4, heads=32, kv_heads=8, head=64, window=1024, lat_heads=32, lat_dim=64,
                               lat_vdim=64, q_rank=768, kv_rank=128, delta_heads=16, delta_kv_heads=8, delta_dim=128, delta_vdim=128,
                               inner=128, ff=8192, vocab=65536)}
    out = {"metric": "Keralix beside Vipotar at equal sizes: prefill of one prompt, decode at batch 8 with 2,048 positions",
           "unit": "tokens/s", "dtype": "bf16", "data": "synthetic (random weights, uniform-random token ids)", "sizes": {}}
    with ClockSampler() as clocks:
        for name, z in sizes.items():
            row = {}
            W, L, F, V = z["width"], z["layers"], z["ff"], z["vocab"]
            for model in ("keralix", "vipotar"):
                if model == "keralix":
                    cfg = keralix_config(**z)
                    n_delta, n_attn = (L + 3) // 4, (L + 2) // 4
                    n_lat = L - n_delta - n_attn
                    H, G, D = z["heads"], z["kv_heads"], z["head"]
                    LH, LD, LV, QR, R = z["lat_heads"], z["lat_dim"], z["lat_vdim"], z["q_rank"], z["kv_rank"]
                    DH, DG, DD, DV, I = z["delta_heads"], z["delta_kv_heads"], z["delta_dim"], z["delta_vdim"], z["inner"]
                    attn = (H + G) * D * W + W * H * D
                    lat = (QR + R + LH * LV) * W + LH * LD * QR + LH * LD * R + LH * LV * R + W * LH * LV
                    delta = (2 * DG * DD + DH * DV + DH + 2 * I) * W + DH * DD * I + DH * DV * I + W * DH * DV
                    matrix = n_attn * attn + n_lat * lat + n_delta * delta + L * 3 * W * F
                    state = n_delta * DH * DD * DV * 4

                    def flops(T):
                        keys = sum(min(t + 1, z["window"]) for t in range(T))
                        return (2.0 * T * matrix + 2.0 * V * W + n_attn * 4.0 * H * D * keys + n_lat * 4.0 * LH * R * T * (T + 1) / 2
                                + n_delta * 7.0 * DH * DD * DV * T)

                    def step_bytes(batch, ctx):
                        per_request = 2 * state + n_attn * min(ctx, z["window"]) * G * D * 2 + n_lat * ctx * R * 2
                        return (matrix + V * W) * 2 + batch * per_request
                    params = matrix + V * W
                else:
                    v = dict(width=W, layers=L, heads=z["heads"], kv_heads=z["kv_heads"], head=z["head"], window=z["window"],
                             lin_heads=z["delta_heads"], lin_dim=z["delta_dim"], lin_vdim=z["delta_vdim"], ff=F, vocab=V)
                    cfg = vipotar_config(**v)
                    qkv = (v["heads"] + 2 * v["kv_heads"]) * v["head"] * W + W * v["heads"] * v["head"]
                    lin = (2 * v["lin_heads"] * v["lin_dim"] + 2 * v["lin_heads"] * v["lin_vdim"]) * W + W * v["lin_heads"] * v["lin_vdim"]
                    matrix = L * (qkv + lin + 2 * W * F)
                    state = L * v["lin_heads"] * v["lin_dim"] * v["lin_vdim"] * 4
                    kv_tok = L * 2 * v["kv_heads"] * v["head"] * 2

                    def flops(T):
                        keys = sum(min(t + 1, v["window"]) for t in range(T))
                        return 2.0 * T * matrix + 2.0 * V * W + L * (4.0 * v["heads"] * v["head"] * keys
                                                                     + 4.0 * v["lin_heads"] * v["lin_dim"] * v["lin_vdim"] * T)

                    def step_bytes(batch, ctx):
                        return (matrix + V * W) * 2 + batch * (2 * state + min(ctx, v["window"]) * kv_tok)
                    params = matrix + 2 * V * W
                engine = Engine(config=cfg, seed=0, dtype="bfloat16", ctx=CTX, parallel=8, page_size=PAGE, max_step_tokens=PROMPT,
                                random_init={"norm_jitter": 0.0})
                r = {"params": params, "prefill": {}}
                for T in (512, 2048):
                    ms = measure_prefill(engine, reps=5, warmup=3, rng=rng, prompt=T)
                    r["prefill"][str(T)] = {"value": round(T * 1000.0 / ms, 1), "ms": round(ms, 3),
                                            "frac": round(flops(T) / (ms * 1e-3) / (pk["bf16_tflops_burst"] * 1e12), 4)}
                ms, launches, library, ctx = measure_decode(engine, 8, max(20, args.steps // 4), max(args.warmup, 3), rng, prompt=PROMPT)
                nbytes = step_bytes(8, ctx)
                r["decode_b8"] = {"value": round(8 * 1000.0 / ms, 1), "ms_per_step": round(ms, 4), "own_kernels_per_step": round(launches, 1),
                                  "library_gemms_per_step": round(library, 1), "bytes_per_step": int(nbytes),
                                  "frac": round(nbytes / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}
                row[model] = r
                del engine
                torch.cuda.empty_cache()
            out["sizes"][name] = dict(row, config=z)
    out["peaks"] = pk["source"]
    out["clocks"] = clocks.summary()
    print(json.dumps(out))
    return 0


def zepesun_config(width, layers, lat_heads, lat_dim, rot_dim, lat_vdim, kv_rank, heads, kv_heads, head, window, mem_heads,
                   mem_dim, mem_vdim, experts, top, groups, keep, ff, vocab, positions):
    """A Zepesun config.json of the given sizes: layers in the order latent attention, parallel (windowed attention beside a
    matrix memory), matrix memory, matrix memory, and so on; the first layer with a dense feed-forward of top * ff features,
    the others routed (`experts` clamped experts of `ff` features in `groups` groups of which `keep` are candidates, `top` per
    token, and a shared one)."""
    lat = {"heads": lat_heads, "dim": lat_dim, "rot_dim": rot_dim, "vdim": lat_vdim, "kv_rank": kv_rank,
           "scale": (lat_dim + rot_dim) ** -0.5, "rot": {"base": 10000.0, "dims": rot_dim}}
    left = {"heads": heads, "kv_heads": kv_heads, "dim": head, "vdim": head, "scale": head ** -0.5, "mask": {"size": window}}
    mem = {"heads": mem_heads, "dim": mem_dim, "vdim": mem_vdim, "gate_cap": 10.0}
    par = {"left": left, "right": mem, "left_scale": 1.0, "right_scale": 1.0}
    moe = {"kind": "moe", "router": {"experts": experts, "top": top, "scale": 2.5, "groups": {"count": groups, "keep": keep}},
           "expert": {"ff": ff, "limit": 7.0}, "shared": {"ff": ff, "limit": 7.0}}
    kinds = [("latent_attention", lat), ("parallel", par), ("mlstm", mem), ("mlstm", mem)]
    return {"architecture": "Zepesun", "vocab": vocab, "width": width, "max_positions": positions, "norm": {"eps": 1e-5},
            "embedding": {"scale": float(width) ** 0.5},
            "layers": [{"type": kinds[i % 4][0], "mixer": kinds[i % 4][1], "mlp": {"kind": "dense", "ff": top * ff} if i == 0 else moe}
                       for i in range(layers)]}


def workload_zepesun(args):
    """Zepesun at two sizes beside Negotar (attention and a gated recurrent mixer in turn, a routed feed-forward: the closest
    design the engine serves) at equal width, depth, attention heads, experts and expert size: prefill of one prompt of 512
    and 2,048 tokens, decode steps of 8 requests with 2,048 positions each.  Rooflines: prefill against the measured
    bfloat16 peak with the flops the design needs (products over all tokens, the experts a token uses and the shared one,
    attention over the window, the latent attention in its latent space over all earlier positions, the matrix memory's
    4 * heads * dim * vdim per token); decode against the measured copy bandwidth with the bytes a step must move (every
    dense matrix once, the experts the step's rows can reach at most and the shared ones, the windows' keys and values, the
    cached latent rows, the memories read and written)."""
    import numpy as np
    import torch
    from imparo_b200.engine import Engine
    rng = np.random.default_rng(0)
    pk = peaks()
    sizes = {"width1024": dict(width=1024, layers=8, lat_heads=16, lat_dim=64, rot_dim=32, lat_vdim=64, kv_rank=96, heads=16, kv_heads=4,
                               head=64, window=512, mem_heads=8, mem_dim=64, mem_vdim=128, experts=16, top=2, groups=4, keep=2, ff=1024,
                               vocab=32768, positions=CTX),
             "width2048": dict(width=2048, layers=8, lat_heads=32, lat_dim=64, rot_dim=32, lat_vdim=64, kv_rank=96, heads=32, kv_heads=8,
                               head=64, window=1024, mem_heads=16, mem_dim=128, mem_vdim=128, experts=32, top=4, groups=8, keep=4, ff=1024,
                               vocab=65536, positions=CTX)}
    out = {"metric": "Zepesun beside Negotar at equal sizes: prefill of one prompt, decode at batch 8 with 2,048 positions",
           "unit": "tokens/s", "dtype": "bf16", "data": "synthetic (random weights, uniform-random token ids)", "sizes": {}}
    with ClockSampler() as clocks:
        for name, z in sizes.items():
            row = {}
            W, L, V = z["width"], z["layers"], z["vocab"]
            expert = 3 * W * z["ff"]
            for model in ("zepesun", "negotar"):
                if model == "zepesun":
                    cfg = zepesun_config(**z)
                    kinds = [cfg["layers"][i]["type"] for i in range(L)]
                    n_lat, n_par = kinds.count("latent_attention"), kinds.count("parallel")
                    n_mem = kinds.count("mlstm") + n_par
                    LH, LD, LR, LV, C = z["lat_heads"], z["lat_dim"], z["rot_dim"], z["lat_vdim"], z["kv_rank"]
                    H, G, D = z["heads"], z["kv_heads"], z["head"]
                    MH, MD, MV = z["mem_heads"], z["mem_dim"], z["mem_vdim"]
                    lat = (LH * (LD + LR) + C + LR + LH) * W + LH * LD * C + LH * LV * C + W * LH * LV
                    left = (2 * H * D + 2 * G * D) * W + W * H * D
                    mem = (2 * MH * MD + 2 * MH * MV + 2 * MH) * W + W * MH * MV
                    dense = n_lat * lat + n_par * left + n_mem * mem + (L - 1) * z["experts"] * W + z["top"] * expert
                    state = n_mem * MH * (MD * MV + MD) * 4

                    def flops(T):
                        keys = sum(min(t + 1, z["window"]) for t in range(T))
                        return (2.0 * T * (dense + (L - 1) * (z["top"] + 1) * expert) + 2.0 * V * W + n_par * 4.0 * H * D * keys
                                + n_lat * 2.0 * LH * (2 * C + LR) * T * (T + 1) / 2 + n_mem * 4.0 * MH * MD * MV * T)

                    def step_bytes(batch, ctx):
                        reached = min(z["experts"], batch * z["top"]) + 1
                        per_request = 2 * state + n_par * min(ctx, z["window"]) * 2 * G * D * 2 + n_lat * ctx * (C + LR) * 2
                        return (dense + (L - 1) * reached * expert + V * W) * 2 + batch * per_request
                    params = dense + (L - 1) * (z["experts"] + 1) * expert + 2 * V * W + z["positions"] * W
                else:
                    n = dict(width=W, layers=L, heads=z["heads"], kv_heads=z["kv_heads"], head=z["head"], ssm_heads=z["mem_heads"] * 2,
                             ssm_vdim=z["mem_vdim"] // 2, ssm_state=z["mem_dim"], experts=z["experts"], top=z["top"], ff=z["ff"], vocab=V)
                    cfg = negotar_config(**n)
                    n_attn = (L + 1) // 2
                    n_ssm = L - n_attn
                    inner, N = n["ssm_heads"] * n["ssm_vdim"], n["ssm_state"]
                    attn = (n["heads"] + 2 * n["kv_heads"]) * n["head"] * W + W * n["heads"] * n["head"]
                    ssm = (2 * inner + 2 * N + n["ssm_heads"]) * W + W * inner
                    dense = n_attn * attn + n_ssm * ssm + L * n["experts"] * W
                    state = n_ssm * n["ssm_heads"] * N * n["ssm_vdim"] * 4
                    kv_tok = n_attn * 2 * n["kv_heads"] * n["head"] * 2
                    params = dense + L * n["experts"] * expert + V * W

                    def flops(T):
                        return (2.0 * T * (dense + L * n["top"] * expert) + 2.0 * V * W
                                + n_attn * 4.0 * n["heads"] * n["head"] * T * (T + 1) / 2 + n_ssm * 6.0 * inner * N * T)

                    def step_bytes(batch, ctx):
                        reached = min(n["experts"], batch * n["top"])
                        return (dense + L * reached * expert + V * W) * 2 + batch * (2 * state + ctx * kv_tok)
                engine = Engine(config=cfg, seed=0, dtype="bfloat16", ctx=CTX, parallel=8, page_size=PAGE, max_step_tokens=PROMPT,
                                random_init={"norm_jitter": 0.0})
                r = {"params": params, "prefill": {}}
                for T in (512, 2048):
                    ms = measure_prefill(engine, reps=5, warmup=3, rng=rng, prompt=T)
                    r["prefill"][str(T)] = {"value": round(T * 1000.0 / ms, 1), "ms": round(ms, 3),
                                            "frac": round(flops(T) / (ms * 1e-3) / (pk["bf16_tflops_burst"] * 1e12), 4)}
                ms, launches, library, ctx = measure_decode(engine, 8, max(20, args.steps // 4), max(args.warmup, 3), rng, prompt=PROMPT)
                nbytes = step_bytes(8, ctx)
                r["decode_b8"] = {"value": round(8 * 1000.0 / ms, 1), "ms_per_step": round(ms, 4), "own_kernels_per_step": round(launches, 1),
                                  "library_gemms_per_step": round(library, 1), "bytes_per_step": int(nbytes),
                                  "frac": round(nbytes / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}
                row[model] = r
                del engine
                torch.cuda.empty_cache()
            out["sizes"][name] = dict(row, config=z)
    out["peaks"] = pk["source"]
    out["clocks"] = clocks.summary()
    print(json.dumps(out))
    return 0


def modinex_config(width, layers, heads, kv_heads, head, vdim, chunk, lin_heads, lin_dim, lin_vdim, ff, vocab, positions):
    """A Modinex config.json of the given sizes: gated linear attention without a feed-forward and attention with one in turn
    (`layers` of each), half of each head rotated, norms in four groups, decays of about 0.9 to 1 per step."""
    rec = {"type": "gla", "mixer": {"heads": lin_heads, "dim": lin_dim, "vdim": lin_vdim, "tau": 16.0, "rank": 16}, "mlp": None}
    att = {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": head, "vdim": vdim, "scale": head ** -0.5,
                                          "mask": {"size": chunk}, "rot": {"dims": head // 2, "base": 500000.0}},
           "mlp": {"kind": "dense", "ff": ff}}
    return {"architecture": "Modinex", "vocab": vocab, "width": width, "max_positions": positions, "norm": {"eps": 1e-6, "groups": 4},
            "layers": [rec, att] * layers}


def workload_modinex(args):
    """Modinex at three sizes beside Vipotar (a grouped-query attention, a linear attention with decay and a dense feed-forward
    per layer: the closest design the engine serves) at equal width, heads, mask size, recurrent state, feed-forward size and
    number of each (a Vipotar layer holds what a pair of Modinex layers holds): prefill of one prompt of 512 and 2,048 tokens,
    decode steps of 8 requests with 2,048 positions each.  Rooflines: prefill against the measured bfloat16 peak with the flops
    the design needs (products over all tokens, attention over what a position sees, the recurrence's 4 * heads * dim * vdim per
    token); decode against the measured copy bandwidth with the bytes a step must move (every matrix once, the keys and values the
    rows see (of a stretch: those since its start), the states read and written)."""
    import numpy as np
    import torch
    from imparo_b200.engine import Engine
    rng = np.random.default_rng(0)
    pk = peaks()
    sizes = {"width1024": dict(width=1024, layers=8, heads=16, kv_heads=4, head=64, window=512, lin_heads=8, lin_dim=64, lin_vdim=128,
                               ff=4096, vocab=32768),
             "width2048": dict(width=2048, layers=8, heads=32, kv_heads=8, head=64, window=1024, lin_heads=16, lin_dim=128, lin_vdim=128,
                               ff=8192, vocab=65536),
             "width2048_head128": dict(width=2048, layers=8, heads=16, kv_heads=4, head=128, window=1024, lin_heads=16, lin_dim=64,
                                       lin_vdim=128, ff=8192, vocab=65536)}
    out = {"metric": "Modinex beside Vipotar at equal sizes: prefill of one prompt, decode at batch 8 with 2,048 positions",
           "unit": "tokens/s", "dtype": "bf16", "data": "synthetic (random weights, uniform-random token ids)", "sizes": {}}
    with ClockSampler() as clocks:
        for name, z in sizes.items():
            row = {}
            W, L, F, V, C = z["width"], z["layers"], z["ff"], z["vocab"], z["window"]
            qkv = (z["heads"] + 2 * z["kv_heads"]) * z["head"] * W + W * z["heads"] * z["head"]
            lin = (2 * z["lin_heads"] * z["lin_dim"] + 2 * z["lin_heads"] * z["lin_vdim"]) * W + W * z["lin_heads"] * z["lin_vdim"]
            state = L * z["lin_heads"] * z["lin_dim"] * z["lin_vdim"] * 4
            kv_tok = L * 2 * z["kv_heads"] * z["head"] * 2
            for model in ("modinex", "vipotar"):
                matrix = L * (qkv + lin + 2 * W * F)
                if model == "modinex":
                    sizes_of = {k: v for k, v in z.items() if k != "window"}
                    cfg = modinex_config(vdim=z["head"], chunk=C, positions=CTX, **sizes_of)
                    matrix += L * (16 * W + z["lin_heads"] * z["lin_dim"] * 16)

                    def keys(T):
                        return sum(t % C + 1 for t in range(T))

                    def step_keys(ctx):
                        return ctx % C
                else:
                    cfg = vipotar_config(**z)

                    def keys(T):
                        return sum(min(t + 1, C) for t in range(T))

                    def step_keys(ctx):
                        return min(ctx, C)

                def flops(T):
                    return (2.0 * T * matrix + 2.0 * V * W + L * 4.0 * z["heads"] * z["head"] * keys(T)
                            + L * 4.0 * z["lin_heads"] * z["lin_dim"] * z["lin_vdim"] * T)

                def step_bytes(batch, ctx):
                    return (matrix + V * W) * 2 + batch * (2 * state + step_keys(ctx) * kv_tok)
                engine = Engine(config=cfg, seed=0, dtype="bfloat16", ctx=CTX, parallel=8, page_size=PAGE, max_step_tokens=PROMPT,
                                random_init={"norm_jitter": 0.0})
                r = {"params": matrix + 2 * V * W, "prefill": {}}
                for T in (512, 2048):
                    ms = measure_prefill(engine, reps=5, warmup=3, rng=rng, prompt=T)
                    r["prefill"][str(T)] = {"value": round(T * 1000.0 / ms, 1), "ms": round(ms, 3),
                                            "frac": round(flops(T) / (ms * 1e-3) / (pk["bf16_tflops_burst"] * 1e12), 4)}
                ms, launches, library, ctx = measure_decode(engine, 8, max(20, args.steps // 4), max(args.warmup, 3), rng, prompt=PROMPT)
                nbytes = step_bytes(8, ctx)
                r["decode_b8"] = {"value": round(8 * 1000.0 / ms, 1), "ms_per_step": round(ms, 4), "own_kernels_per_step": round(launches, 1),
                                  "library_gemms_per_step": round(library, 1), "bytes_per_step": int(nbytes),
                                  "frac": round(nbytes / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}
                row[model] = r
                del engine
                torch.cuda.empty_cache()
            out["sizes"][name] = dict(row, config=z)
    out["peaks"] = pk["source"]
    out["clocks"] = clocks.summary()
    print(json.dumps(out))
    return 0


def zinunex_config(width, layers, lat_heads, lat_dim, rot_dim, lat_vdim, kv_rank, heads, kv_heads, head, window, experts, top, groups, keep,
                   ff, side, vocab):
    """A Zinunex config.json of the given sizes: per four layers a windowed latent attention, two attentions and a latent attention
    that reads the first one's cache; a routed feed-forward with a shared expert of the experts' size everywhere."""
    rot = {"base": 500000.0, "dims": rot_dim, "scaling": {"factor": 4.0, "original": 2048, "fast": 32.0, "slow": 1.0}}
    lat = {"heads": lat_heads, "dim": lat_dim, "rot_dim": rot_dim, "vdim": lat_vdim, "kv_rank": kv_rank, "scale": (lat_dim + rot_dim) ** -0.5,
           "mask": {"size": window}, "rot": rot}
    att = {"heads": heads, "kv_heads": kv_heads, "dim": head, "vdim": head, "scale": head ** -0.5,
           "rot": {"base": 500000.0, "dims": head, "scaling": {"factor": 4.0}}}
    moe = {"kind": "moe", "router": {"experts": experts, "top": top, "scale": 2.0, "groups": {"count": groups, "keep": keep}},
           "expert": {"ff": ff}, "shared": {"ff": ff}}
    kinds = []
    for i in range(0, layers, 4):
        kinds += [("latent_attention", lat), ("attention", att), ("attention", att), ("latent_attention", dict(lat, kv_from=i))]
    return {"architecture": "Zinunex", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "token_side": {"dim": side},
            "layers": [{"type": t, "mixer": m, "mlp": moe} for t, m in kinds[:layers]]}


def workload_zinunex(args):
    """Zinunex at three sizes beside Zepesun (whose latent attention, grouped router and shared expert are the closest the engine
    serves) at equal width, depth, latent heads and cached rows, experts and parameters per expert (two matrices of 1.5 ff features
    beside three of ff): every Zepesun layer a latent attention with a routed feed-forward; every second pair of Zinunex layers an
    attention of as many heads instead.  Prefill of one prompt of 512 and 2,048 tokens, decode steps of 8 requests with 2,048
    positions each.  Rooflines: prefill against the measured bfloat16 peak with the flops the design needs (products over all tokens,
    the experts a token uses and the shared one, attention over the keys a position sees, the latent attention in its latent space);
    decode against the measured copy bandwidth with the bytes a step must move (every dense matrix once, the experts the step's
    rows can reach at most and the shared ones, the cached keys and values or latent rows the rows see, the tokens' side entries)."""
    import numpy as np
    import torch
    from imparo_b200.engine import Engine
    rng = np.random.default_rng(0)
    pk = peaks()
    sizes = {"width1024": dict(width=1024, layers=8, lat_heads=16, lat_dim=64, rot_dim=32, lat_vdim=64, kv_rank=96, heads=16, kv_heads=4,
                               head=64, window=512, experts=16, top=2, groups=4, keep=2, ff=1536, side=128, vocab=32768),
             "width2048": dict(width=2048, layers=8, lat_heads=32, lat_dim=64, rot_dim=32, lat_vdim=64, kv_rank=96, heads=32, kv_heads=8,
                               head=64, window=1024, experts=32, top=4, groups=8, keep=4, ff=1536, side=256, vocab=65536),
             "width2048_head128": dict(width=2048, layers=8, lat_heads=16, lat_dim=128, rot_dim=32, lat_vdim=128, kv_rank=96, heads=16,
                                       kv_heads=4, head=128, window=1024, experts=16, top=2, groups=4, keep=2, ff=3072, side=256, vocab=65536)}
    if args.only_size:
        sizes = {k: v for k, v in sizes.items() if k == args.only_size}
    out = {"metric": "Zinunex beside Zepesun at equal sizes: prefill of one prompt, decode at batch 8 with 2,048 positions",
           "unit": "tokens/s", "dtype": "bf16", "data": "synthetic (random weights, uniform-random token ids)", "sizes": {}}
    with ClockSampler() as clocks:
        for name, z in sizes.items():
            row = {}
            W, L, V, S = z["width"], z["layers"], z["vocab"], z["side"]
            LH, LD, LR, LV, C = z["lat_heads"], z["lat_dim"], z["rot_dim"], z["lat_vdim"], z["kv_rank"]
            H, G, D = z["heads"], z["kv_heads"], z["head"]
            expert = 2 * W * z["ff"]
            for model in ("zinunex", "zepesun"):
                lat = LH * (LD + LR) * W + LH * (LD + LV) * C + W * LH * LV          # without the latent's own projection
                if model == "zinunex":
                    cfg = zinunex_config(**z)
                    n_lat = sum(e["type"] == "latent_attention" for e in cfg["layers"])
                    n_own = sum("kv_from" not in e["mixer"] for e in cfg["layers"] if e["type"] == "latent_attention")
                    n_att, window = L - n_lat, z["window"]
                    dense = (n_lat * lat + n_own * (C + LR) * W + n_att * ((2 * H + G) * D * W) + L * (z["experts"] + 1) * W + L * 2 * S * W)
                    side = L * S
                else:
                    cfg = zepesun_config(width=W, layers=L, lat_heads=LH, lat_dim=LD, rot_dim=LR, lat_vdim=LV, kv_rank=C, heads=H, kv_heads=G,
                                         head=D, window=z["window"], mem_heads=1, mem_dim=8, mem_vdim=8, experts=z["experts"], top=z["top"],
                                         groups=z["groups"], keep=z["keep"], ff=z["ff"] * 2 // 3, vocab=V, positions=CTX)
                    first, moe = cfg["layers"][0], cfg["layers"][1]["mlp"]
                    cfg["layers"] = [dict(first, mlp=moe) for _ in range(L)]
                    n_lat = n_own = L
                    n_att, window, side = 0, None, 0
                    dense = L * (lat + (C + LR + LH) * W) + L * z["experts"] * W

                def flops(T):
                    keys = sum(min(t + 1, window or T) for t in range(T))
                    return (2.0 * T * (dense + L * (z["top"] + 1) * expert) + 2.0 * V * W + n_att * 4.0 * H * D * T * (T + 1) / 2
                            + n_lat * 2.0 * LH * (2 * C + LR) * keys)

                def step_bytes(batch, ctx):
                    reached = min(z["experts"], batch * z["top"]) + 1
                    # (a layer that reads another one's cached rows reads them again)
                    per_request = n_att * ctx * 2 * G * D * 2 + n_lat * min(ctx, window or ctx) * (C + LR) * 2 + side * 2
                    return (dense + L * reached * expert + V * W) * 2 + batch * per_request
                params = dense + L * (z["experts"] + 1) * expert + 2 * V * W + V * side + (CTX * W if model == "zepesun" else 0)
                engine = Engine(config=cfg, seed=0, dtype="bfloat16", ctx=CTX, parallel=8, page_size=PAGE, max_step_tokens=PROMPT,
                                random_init={"norm_jitter": 0.0})
                r = {"params": params, "prefill": {}}
                for T in (512, 2048):
                    ms = measure_prefill(engine, reps=5, warmup=3, rng=rng, prompt=T)
                    r["prefill"][str(T)] = {"value": round(T * 1000.0 / ms, 1), "ms": round(ms, 3),
                                            "frac": round(flops(T) / (ms * 1e-3) / (pk["bf16_tflops_burst"] * 1e12), 4)}
                ms, launches, library, ctx = measure_decode(engine, 8, max(20, args.steps // 4), max(args.warmup, 3), rng, prompt=PROMPT)
                nbytes = step_bytes(8, ctx)
                r["decode_b8"] = {"value": round(8 * 1000.0 / ms, 1), "ms_per_step": round(ms, 4), "own_kernels_per_step": round(launches, 1),
                                  "library_gemms_per_step": round(library, 1), "bytes_per_step": int(nbytes),
                                  "frac": round(nbytes / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4)}
                row[model] = r
                del engine
                torch.cuda.empty_cache()
            out["sizes"][name] = dict(row, config=z)
    out["peaks"] = pk["source"]
    out["clocks"] = clocks.summary()
    print(json.dumps(out))
    return 0


def _preset(name):
    with open(os.path.join(ROOT, "imparo_b200", "config", "presets", name + ".json")) as f:
        return json.load(f)


def workload_continuous(args):
    """LFM2-700M sizes: a continuous batch of requests (32 unless --requests says otherwise) with prompt lengths
    uniform in [64, 4096] through 32 slots, prompts in portions under a 512-token step budget beside the running
    decode rows, temperature 0.7 (seeded), 128 new tokens each; requests join and leave mid-run, and with more
    requests than slots, slots and pages are used again.  Besides tokens per second: the step-time split (the
    reference prints step / gpu / gap medians for its loop, imparo-server/src/sched.rs:572-649): per class of step
    (decode rows only; portions beside decode rows; portions only) the device time between the events recorded after
    consecutive steps, the host time between their launches, and, for steps of decode rows only, the bytes they have
    to read (weights once, the cache of their rows) over that time against the measured HBM peak."""
    import numpy as np
    import torch
    from imparo_b200.engine import Engine
    from imparo_b200.kernels import ops
    rng = np.random.default_rng(1)
    n, slots, new = args.requests, 32, 128
    engine = Engine(config=_preset("lfm2_700m"), seed=0, dtype="bfloat16", ctx=4096 + new, parallel=slots, page_size=PAGE,
                    max_step_tokens=512, random_init={"norm_jitter": 0.0})
    pk = peaks()
    weight_bytes, kv_per_token, prefill_flops, n_params = model_numbers(engine)
    V = engine.vocab_size
    lens = [int(x) for x in rng.integers(64, 4097, n)]
    prompts = [rng.integers(0, V, k).tolist() for k in lens]
    engine.generate(prompts[:4], max_tokens=8, temperature=0.7, seed=list(range(4)))       # warm-up: buffers, first graphs
    steps = []                # per step: (class, event after it, host time, bytes of a decode-only step, tokens)

    def on_step(plan):
        portions = any(e.count > 1 or e.start == 0 for e in plan)
        rows = any(e.count == 1 and e.start > 0 for e in plan)
        kind = "portions_beside_decode_rows" if portions and rows else ("portions_only" if portions else "decode_rows_only")
        ev = torch.cuda.Event(enable_timing=True)
        ev.record()
        nbytes = weight_bytes + kv_per_token * sum(e.start + e.count for e in plan)
        steps.append((kind, ev, time.perf_counter(), nbytes, sum(e.count for e in plan), len(plan)))
    # Two passes over the same requests with the same engine.  The first meets every step shape for the first time
    # (a new shape runs launch by launch once and is captured the second time it comes); the second is the timed
    # one: a server in its steady state, whose shapes have come before.  Both are reported.
    first = {}
    for timed in (False, True):
        steps.clear()
        before, replays, captures = dict(ops.COUNTS), engine.step_fn.graph_replays, engine.step_fn.graph_captures
        with ClockSampler() as clocks:
            t0 = time.perf_counter()
            out = engine.generate(prompts, max_tokens=new, temperature=0.7, seed=list(range(n)), on_step=on_step, stop_token_ids=[])
            torch.cuda.synchronize()
            dt = time.perf_counter() - t0
        assert all(len(o) == new for o in out)
        if not timed:
            first = {"value": round((sum(lens) + n * new) / dt, 1), "seconds": round(dt, 3), "steps": len(steps),
                     "graph_replays": engine.step_fn.graph_replays - replays,
                     "graph_captures": engine.step_fn.graph_captures - captures}
    st = engine.stats()
    split = {}
    for kind in ("decode_rows_only", "portions_beside_decode_rows", "portions_only"):
        dev, host, gbs, toks = [], [], [], []
        for i in range(1, len(steps)):
            if steps[i][0] != kind:
                continue
            d_ms = steps[i - 1][1].elapsed_time(steps[i][1])
            dev.append(d_ms)
            host.append((steps[i][2] - steps[i - 1][2]) * 1e3)
            toks.append(steps[i][4])
            if kind == "decode_rows_only" and d_ms > 0:
                gbs.append(steps[i][3] / (d_ms * 1e-3) / 1e9)
        if dev:
            split[kind] = {"steps": len(dev), "device_ms_median": round(statistics.median(dev), 4),
                           "host_ms_between_launches_median": round(statistics.median(host), 4),
                           "tokens_per_step_mean": round(sum(toks) / len(toks), 1)}
            if gbs:
                split[kind]["roofline"] = {"bound": "hbm", "achieved": round(statistics.median(gbs), 1), "peak": pk["hbm_gbs"],
                                           "unit": "GB/s", "frac": round(statistics.median(gbs) / pk["hbm_gbs"], 4),
                                           "peaks": pk["source"]}
    device_total = steps[0][1].elapsed_time(steps[-1][1]) * 1e-3 if len(steps) > 1 else 0.0
    flops = sum(prefill_flops(k) for k in lens)
    print(json.dumps({
        "metric": "LFM2-700M continuous batching, prompt + generated tokens per second (wall clock, through Engine.generate)",
        "value": round((sum(lens) + n * new) / dt, 1), "unit": "tokens/s", "generated_per_s": round(n * new / dt, 1),
        "seconds": round(dt, 3), "device_seconds_first_to_last_step": round(device_total, 3),
        "requests": n, "slots": slots, "prompt_tokens": sum(lens), "new_tokens": n * new,
        "first_pass": first, "step_budget": 512, "steps": len(steps), "mean_rows_per_step": round(sum(s_[5] for s_ in steps) / max(len(steps), 1), 1),
        "step_time_split": split,
        "prompt_flops_over_time_frac_of_bf16_peak": round(flops / max(dt, 1e-9) / (pk["bf16_tflops"] * 1e12), 4),
        "graph_replays": engine.step_fn.graph_replays - replays, "graph_captures": engine.step_fn.graph_captures - captures,
        "graph_resets": engine.step_fn.graph_resets, "preemptions": st["preemptions"], "failed": st["failed"],
        "own_kernel_launches": ops.COUNTS["own"] - before["own"], "library_gemms": ops.COUNTS["library"] - before["library"],
        "dtype": "bf16", "data": "synthetic (random weights, uniform-random token ids)", "clocks": clocks.summary()}))
    return 0


def workload_long(args):
    """LFM2-350M sizes: 4 requests with 32,768-token prompts and 512 greedy tokens each, in bfloat16 (all 16 layers:
    throughput, with the prefill's flops over its time against the measured bfloat16 peak and the decode step's bytes
    over its time against the measured HBM peak).  Then the 32-bit check: the logits at sampled positions of one
    32,768-token prompt, through the engine whole and in portions of 1,024 tokens, against the plain implementation
    (tests/plain, numpy, whole sequence, no cache).  The plain forward over 32,768 tokens is slow, so the check runs
    on the first --long-check-layers layers of the configuration (4 by default: two convolution blocks and two
    attention blocks, every width as configured); `config` names both numbers."""
    import tempfile
    import numpy as np
    import torch
    from imparo_b200.engine import Engine, StepItem
    from imparo_b200.weights import write_random_model
    cfg = _preset("lfm2_350m")
    pk = peaks()
    rng = np.random.default_rng(2)
    P, new, B = 32768, 512, 4
    out = {"metric": "LFM2-350M long context: 4 x 32,768-token prompts + 512 greedy tokens", "unit": "tokens/s",
           "data": "synthetic (random weights, uniform-random token ids)", "dtype": "bf16 (throughput), fp32 (check)"}
    engine = Engine(config=cfg, seed=0, dtype="bfloat16", ctx=P + new, parallel=B, page_size=PAGE, max_step_tokens=P,
                    random_init={"norm_jitter": 0.0})
    weight_bytes, kv_per_token, prefill_flops, n_params = model_numbers(engine)
    prompts = [rng.integers(0, engine.vocab_size, P).tolist() for _ in range(B)]
    stamps = []

    def on_step(plan):
        ev = torch.cuda.Event(enable_timing=True)
        ev.record()
        stamps.append((time.perf_counter(), sum(e.count for e in plan), ev))
    # a first pass of the same shapes (buffers sized, the prompt step and the decode step captured), timed apart
    torch.cuda.synchronize()
    t0 = time.perf_counter()
    engine.generate(prompts, max_tokens=16, stop_token_ids=[], on_step=on_step)
    torch.cuda.synchronize()
    first_decode = next(i for i, (_, c, _) in enumerate(stamps) if c == B)
    out["first_pass"] = {"prefill_tokens_per_s": round(B * P / (stamps[first_decode][0] - t0), 1),
                         "prefill_ms": round((stamps[first_decode][0] - t0) * 1e3, 1)}
    stamps.clear()
    with ClockSampler() as clocks:
        t0 = time.perf_counter()
        got = engine.generate(prompts, max_tokens=new, stop_token_ids=[], on_step=on_step)
        torch.cuda.synchronize()
        dt = time.perf_counter() - t0
    assert all(len(g) == new for g in got)
    first_decode = next(i for i, (_, c, _) in enumerate(stamps) if c == B)
    prefill_s = stamps[first_decode][0] - t0
    decode = [stamps[i - 1][2].elapsed_time(stamps[i][2]) for i in range(first_decode + 1, len(stamps)) if stamps[i][1] == B]
    dec_ms = statistics.median(decode)
    step_bytes = weight_bytes + B * (P + new / 2) * kv_per_token
    out["value"] = round(B * P / prefill_s, 1)
    out["bf16"] = {"seconds": round(dt, 3), "prefill_tokens_per_s": round(B * P / prefill_s, 1),
                   "prefill": {"tokens": B * P, "ms": round(prefill_s * 1e3, 1),
                               "frac": round(B * prefill_flops(P) / prefill_s / (pk["bf16_tflops"] * 1e12), 4)},
                   "decode_tokens_per_s": round(B * 1000.0 / dec_ms, 1), "decode_ms_per_step": round(dec_ms, 4),
                   "roofline": {"bound": "hbm", "achieved": round(step_bytes / (dec_ms * 1e-3) / 1e9, 1), "peak": pk["hbm_gbs"],
                                "unit": "GB/s", "frac": round(step_bytes / (dec_ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4),
                                "peaks": pk["source"], "bytes_per_step": int(step_bytes)},
                   "new_tokens_each": new, "layers": cfg["num_hidden_layers"]}
    del engine
    torch.cuda.empty_cache()

    # ---- the 32-bit check against the plain implementation ----
    from tests.plain.lfm2_plain import PlainLfm2
    n_layers = args.long_check_layers
    small = dict(cfg)
    # the configuration's first blocks up to and including its second attention block, cut to n_layers by keeping the
    # last n_layers of them: two convolution and two attention blocks at the default of 4
    types = list(cfg["layer_types"])
    second_attn = [i for i, t_ in enumerate(types) if t_ != "conv"][1]
    small["layer_types"] = types[max(0, second_attn + 1 - n_layers):second_attn + 1] if n_layers < len(types) else types
    small["num_hidden_layers"] = len(small["layer_types"])
    places = [0, 1023, 1024, 16384, P - 1]
    toks = prompts[0]
    with tempfile.TemporaryDirectory(prefix="imparo_b200_long_") as d:
        write_random_model(d, small, seed=0, dtype="float32", norm_jitter=0.1)
        t1 = time.perf_counter()
        ref = PlainLfm2(d, np.float32).logits_at(toks, places, attend_block=256).astype(np.float64)
        plain_s = time.perf_counter() - t1
        engine = Engine(d, dtype="float32", ctx=P, parallel=1, page_size=PAGE, max_step_tokens=P)
        rows = {}
        for name, cut in (("whole", P), ("portions_of_1024", 1024)):
            engine.add_request(900 + cut)
            got_rows, at = [], 0
            t2 = time.perf_counter()
            while at < P:
                k = min(cut, P - at)
                want = [p_ - at for p_ in places if at <= p_ < at + k]
                lg = engine.step([StepItem(900 + cut, toks[at:at + k], want)])
                if want:
                    got_rows.append(lg.double().cpu().numpy())
                at += k
            torch.cuda.synchronize()
            rows[name] = (np.concatenate(got_rows), time.perf_counter() - t2)
            engine.end_request(900 + cut)
        engine.check_device_status()
    scale = float(np.abs(ref).max())
    out["fp32"] = {"layers": small["num_hidden_layers"], "layers_of_config": cfg["num_hidden_layers"],
                   "layer_types": small["layer_types"], "positions": places, "logit_scale": round(scale, 4),
                   "vs_plain_max_abs_diff": {k: float(np.abs(v[0] - ref).max()) for k, v in rows.items()},
                   "vs_plain_max_abs_diff_over_scale": {k: float(np.abs(v[0] - ref).max() / scale) for k, v in rows.items()},
                   "whole_vs_portions_max_abs_diff": float(np.abs(rows["whole"][0] - rows["portions_of_1024"][0]).max()),
                   "same_argmax_as_plain": {k: bool((v[0].argmax(-1) == ref.argmax(-1)).all()) for k, v in rows.items()},
                   "engine_seconds": {k: round(v[1], 2) for k, v in rows.items()}, "plain_seconds": round(plain_s, 1),
                   "plain": "tests/plain/lfm2_plain.py, numpy float32, whole sequence, attention a block of 256 queries at a time"}
    out["vs_plain_max_abs_diff"] = max(out["fp32"]["vs_plain_max_abs_diff"].values())
    out["config"] = {"model": "LFM2-350M", "global_batch": B, "prompt_len": P, "new_tokens": new, "layers": cfg["num_hidden_layers"],
                     "layers_of_config": cfg["num_hidden_layers"], "check_layers": small["num_hidden_layers"],
                     "hidden": cfg["hidden_size"], "heads": cfg["num_attention_heads"], "kv_heads": cfg["num_key_value_heads"],
                     "vocab": cfg["vocab_size"], "page_size": PAGE, "params": n_params}
    out["clocks"] = clocks.summary()
    print(json.dumps(out))
    return 0


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=256)
    ap.add_argument("--warmup", type=int, default=20)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--layers", type=int, default=None, help="run fewer layers than the configuration has (named in config)")
    ap.add_argument("--skip-points", action="store_true", help="skip the batch-1 and batch-64 points")
    ap.add_argument("--only-decode", action="store_true", help="time the decode steps only (for profiler captures)")
    ap.add_argument("--only-prefill", action="store_true", help="time the 2,048-token prompt only (for profiler captures)")
    ap.add_argument("--workload", default="headline", choices=["headline", "continuous", "long", "sizes", "vipotar", "negotar", "keralix", "zepesun", "modinex", "zinunex"],
                    help="headline (default): the one JSON line described at the top of this file.  continuous: LFM2-700M sizes, requests with prompts "
                         "of 64 to 4,096 tokens through 32 slots in 512-token portions beside decode rows, temperature 0.7, 128 new "
                         "tokens each.  long: LFM2-350M sizes, 4 prompts of 32,768 tokens and 512 greedy tokens each, bfloat16 and 32-bit.  "
                         "vipotar / negotar: that design at two sizes beside LFM2 at equal sizes.  keralix: the Keralix design at two sizes beside Vipotar")
    ap.add_argument("--only-size", default=None, help="zinunex: run one of the sizes")
    ap.add_argument("--requests", type=int, default=32, help="continuous: requests in all (the baseline's workload has 32)")
    ap.add_argument("--long-check-layers", type=int, default=4, help="long: layers of the 32-bit check against the plain implementation")
    args = ap.parse_args()
    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable": "zeraix/imparo is a Rust workspace (no setup.py or pyproject.toml: "
                          "pip reports 'not installable') and this image has no cargo/rustc, so it cannot be built or run here"}))
        return 0
    if args.gpus != 1:
        print("bench.py: this engine runs on ONE GPU; --gpus > 1 is not supported (nothing was measured)")
        return 2
    import numpy as np
    import torch
    from imparo_b200.engine import Engine
    from imparo_b200.kernels import ops

    if args.workload == "continuous":
        return workload_continuous(args)
    if args.workload == "long":
        return workload_long(args)
    if args.workload == "sizes":
        return workload_sizes(args)
    if args.workload == "vipotar":
        return workload_vipotar(args)
    if args.workload == "negotar":
        return workload_negotar(args)
    if args.workload == "keralix":
        return workload_keralix(args)
    if args.workload == "zepesun":
        return workload_zepesun(args)
    if args.workload == "modinex":
        return workload_modinex(args)
    if args.workload == "zinunex":
        return workload_zinunex(args)
    cfg = dict(LFM2_1_2B)
    if args.layers is not None and args.layers < cfg["num_hidden_layers"]:
        cfg["layer_types"] = cfg["layer_types"][:args.layers]
        cfg["num_hidden_layers"] = args.layers
    steps, warmup = args.steps, max(args.warmup, 3)
    rng = np.random.default_rng(0)
    max_batch = args.batch if (args.skip_points or args.only_decode or args.only_prefill) else max(64, args.batch)
    engine = Engine(config=cfg, seed=0, dtype="bfloat16", ctx=CTX, parallel=max_batch, page_size=PAGE,
                    max_step_tokens=PROMPT, random_init={"norm_jitter": 0.0})
    pk = peaks()
    weight_bytes, kv_per_token, prefill_flops, n_params = model_numbers(engine)

    if args.only_prefill:
        pre_ms = measure_prefill(engine, reps=max(1, steps), warmup=warmup, rng=rng)
        print(json.dumps({"metric": "prefill only", "tokens": PROMPT, "ms": round(pre_ms, 3),
                          "value": round(PROMPT * 1000.0 / pre_ms, 1),
                          "frac": round(prefill_flops(PROMPT) / (pre_ms * 1e-3) / (pk["bf16_tflops_burst"] * 1e12), 4)}))
        return 0
    with ClockSampler() as clocks:
        ms, launches, library, ctx = measure_decode(engine, args.batch, steps, warmup, rng)
    value = args.batch * 1000.0 / ms
    step_bytes = weight_bytes + args.batch * ctx * kv_per_token
    achieved = step_bytes / (ms * 1e-3) / 1e9

    if args.only_decode:
        print(json.dumps({"metric": "decode only", "batch": args.batch, "ms_per_step": round(ms, 4), "value": round(value, 1),
                          "achieved_gbs": round(achieved, 1), "own_kernels_per_step": launches, "library_gemms_per_step": library}))
        return 0
    pre_ms = measure_prefill(engine, reps=5, warmup=3, rng=rng)
    pre_flops = prefill_flops(PROMPT)
    prefill = {"value": round(PROMPT * 1000.0 / pre_ms, 1), "tokens": PROMPT, "ms": round(pre_ms, 3),
               "frac": round(pre_flops / (pre_ms * 1e-3) / (pk["bf16_tflops_burst"] * 1e12), 4)}

    points = {}
    if not args.skip_points:
        for b in (1, 64):
            pms, _, _, _ = measure_decode(engine, b, max(20, steps // 4), warmup, rng)
            points[f"decode_b{b}"] = round(b * 1000.0 / pms, 1)

    # h2d: the step's descriptor (tokens, positions, request index, row starts, slots, start
    # positions, wanted rows, one block-table row per request), counted from the copied tensor
    e2e_value, h2d = measure_e2e(engine, args.batch, steps, warmup, rng)

    line = {
        "metric": "LFM2-1.2B decode tok/s @ batch 8 (2,048-token prompts, ctx 4,096)", "value": round(value, 1), "unit": "tokens/s",
        "n_gpus": 1, "steps": steps, "warmup": warmup, "ms_per_step": round(ms, 4), "higher_is_better": True,
        "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic (random weights, uniform-random token ids)",
        "impl": "ours",
        "config": {"model": "LFM2-1.2B", "global_batch": args.batch, "seq_len": CTX, "prompt_len": PROMPT, "parallelism": "1gpu",
                   "layers": cfg["num_hidden_layers"], "layers_of_config": LFM2_1_2B["num_hidden_layers"],
                   "hidden": cfg["hidden_size"], "heads": 32, "kv_heads": 8, "head_dim": 64, "ff_dim": engine.config.ff_dim,
                   "vocab": cfg["vocab_size"], "conv_L_cache": 3, "page_size": PAGE, "params": n_params,
                   "l2": "inputs larger than L2 (2.3 GB of weights read per step)", "cuda_graph": True,
                   "last_ffn": "wanted rows only"},
        "e2e": {"value": round(e2e_value, 1), "unit": "tokens/s", "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": 4 * args.batch},
        "gpu_launches": int(round(launches * steps)), "own_kernels_per_step": round(launches, 1),
        "library_gemms_per_step": round(library, 1),
        "prefill": prefill,
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4), "peaks": pk["source"], "bytes_per_step": int(step_bytes)},
        "points": points,
        "clocks": clocks.summary(),
    }
    print(json.dumps(line))
    return 0


if __name__ == "__main__":
    sys.exit(main())
