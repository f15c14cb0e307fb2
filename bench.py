#!/usr/bin/env python3
"""Decode and prefill throughput at Qwen3-8B layer sizes, random bf16 weights.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--layers L] [--impl ours|reference]
                    [--arms 8b,14b,32b]

A "step" is one decode step of a batch of 8 sequences (512-token prompts, the
cache sized for a context of 4,096 per sequence).  W untimed decode steps, then
exactly K timed ones between CUDA events with a synchronize on both sides.
The weights (15 GB a step) are far larger than L2, so nothing is flushed
between steps.  Prints ONE JSON line.

Beside the headline the line holds: `e2e` (the same through the Python entry
point, host tokens in and out), `prefill` (one 2,048-token prompt), `points`
(decode at batch 1 and 64 over 256 steps from 512-token prompts, whatever
--steps is; and, unless --arms leaves them out, the two larger workloads: at
Qwen3-14B sizes 16 prompts of seeded lengths in [64, 2048] and 128 steps
sampled at temperature 0.7 through the entry point; at Qwen3-32B sizes batch 32
from 1,024-token prompts over 256 steps and one 8,192-token prefill, the cache
sized to 8,192 a slot), `points_frac` (each point's fraction of its roofline)
and `finite` (every logit of the last timed step is a finite number).
"""

import argparse
import json
import os
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

QWEN3_8B = {
    "architectures": ["Qwen3ForCausalLM"], "model_type": "qwen3",
    "num_hidden_layers": 36, "hidden_size": 4096, "num_attention_heads": 32,
    "num_key_value_heads": 8, "head_dim": 128, "intermediate_size": 12288, "vocab_size": 151936,
    "rope_theta": 1000000.0, "rms_norm_eps": 1e-6, "tie_word_embeddings": False,
    "max_position_embeddings": 40960, "hidden_act": "silu", "attention_bias": False,
    "rope_scaling": None, "use_sliding_window": False, "sliding_window": None,
}
# the other sizes of the family, for runs beyond the default (--shape)
SHAPES = {
    "8b": {},
    "14b": {"num_hidden_layers": 40, "hidden_size": 5120, "num_attention_heads": 40, "intermediate_size": 17408},
    "32b": {"num_hidden_layers": 64, "hidden_size": 5120, "num_attention_heads": 64, "intermediate_size": 25600},
}
CONTEXT = 4096
PROMPT = 512
PREFILL_TOKENS = 2048
POINT_STEPS = 256  # decode steps of the batch 1 / 64 / 32 points: contexts 512 -> 768, as the workload is stated


def peaks():
    p = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        with open(path) as f:
            m = json.load(f)
        p = {"hbm_gbs": float(m["hbm_gbs"]), "bf16_tflops": float(m["bf16_tflops"]), "source": "measured"}
    return p


class ClockSampler:
    """nvidia-smi clocks and throttle reasons during the timed region."""

    Q = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,"
         "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
         "clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.samples = []
        self.proc = None

    def start(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", "-i", "0", f"--query-gpu={self.Q}", "--format=csv,noheader,nounits", "-lms", "100"],
                stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.samples.append((time.time(), line.strip()))

    def mark(self):
        return time.time()

    def stop(self):
        if self.proc is not None:
            self.proc.terminate()

    def summary(self, t0, t1):
        sm, mx, reasons = [], 0, set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for t, line in self.samples:
            if not (t0 - 0.05 <= t <= t1 + 0.15):
                continue
            parts = [x.strip() for x in line.split(",")]
            try:
                sm.append(float(parts[0]))
                mx = max(mx, float(parts[1]))
            except (ValueError, IndexError):
                continue
            for n, v in zip(names, parts[2:6]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        sm.sort()
        return {"sm_mhz": sm[len(sm) // 2] if sm else None, "sm_max_mhz": mx or None,
                "samples": len(sm), "reasons": sorted(reasons)}


def model_numbers(cfg, layers):
    H, I, V = cfg["hidden_size"], cfg["intermediate_size"], cfg["vocab_size"]
    nq, nkv, d = cfg["num_attention_heads"], cfg["num_key_value_heads"], cfg["head_dim"]
    per_layer = H * (nq + 2 * nkv) * d + nq * d * H + 3 * H * I
    weight_bytes = 2 * (layers * per_layer + V * H)  # every matrix a decode step reads, bf16
    kv_bytes_per_token = layers * 2 * nkv * d * 2
    return per_layer, weight_bytes, kv_bytes_per_token


def prefill_flops(cfg, layers, T):
    per_layer, _, _ = model_numbers(cfg, layers)
    nq, d = cfg["num_attention_heads"], cfg["head_dim"]
    gemm = 2.0 * T * (layers * per_layer + cfg["vocab_size"] * cfg["hidden_size"] * (1.0 / T))
    attn = layers * nq * 2.0 * T * T * d  # causal: QK^T and PV, half of the square each
    return gemm + attn


class Arm:
    """One model size on the device with its engine; freed before the next."""

    def __init__(self, shape, layers, max_tokens, max_batch):
        import torch

        from reflex_b200.api import Model
        from reflex_b200.weights import random_model_on_device

        cfg = dict(QWEN3_8B)
        cfg.update(SHAPES[shape])
        self.full_layers = cfg["num_hidden_layers"]
        self.layers = layers or self.full_layers
        cfg["num_hidden_layers"] = self.layers
        self.cfg, self.shape = cfg, shape
        lm = random_model_on_device(cfg, 0, torch.bfloat16, "cuda:0")
        self.model = Model(lm, max_tokens=max_tokens, max_batch=max_batch)
        self.eng = self.model.engine
        self.V = cfg["vocab_size"]
        self.g = torch.Generator().manual_seed(1)
        _, self.weight_bytes, self.kv_per_tok = model_numbers(cfg, self.layers)

    def free(self):
        import gc

        import torch

        self.model = self.eng = None
        gc.collect()
        torch.cuda.empty_cache()

    def decode_run(self, batch, prompt_len, steps, warmup, sampler=None):
        """Prefill `batch` prompts of `prompt_len` tokens, then warmup + steps
        greedy decode steps fed from the device; returns a dict."""
        import torch

        from reflex_b200 import ops

        eng = self.eng
        prompts = torch.randint(0, self.V, (batch, prompt_len), generator=self.g).tolist()
        seqs = [eng.open() for _ in range(batch)]
        logits = eng.step([(s, p, [prompt_len - 1]) for s, p in zip(seqs, prompts)])
        # the picked ids stay on the device and feed the next step (two buffers in turn)
        ids = [torch.empty((batch,), dtype=torch.int32, device="cuda:0") for _ in range(2)]
        scratch = torch.empty((batch * 128,), dtype=torch.float32, device="cuda:0")
        ops.argmax(logits, out=ids[0], scratch=scratch)
        for i in range(warmup):
            logits = eng.step_decode(seqs, ids[i % 2], borrow=True)
            ops.argmax(logits, out=ids[(i + 1) % 2], scratch=scratch)
        ctx0 = eng.length(seqs[0])
        start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        t0 = sampler.mark() if sampler else 0
        start.record()
        for i in range(warmup, warmup + steps):
            logits = eng.step_decode(seqs, ids[i % 2], borrow=True)
            ops.argmax(logits, out=ids[(i + 1) % 2], scratch=scratch)
        end.record()
        torch.cuda.synchronize()
        t1 = sampler.mark() if sampler else 0
        finite = bool(torch.isfinite(logits).all().item())  # after the timed region
        eng.check_errors()
        ms = start.elapsed_time(end) / steps
        mean_ctx = ctx0 + (steps + 1) / 2.0
        for s in seqs:
            eng.close(s)
        bytes_step = self.weight_bytes + batch * mean_ctx * self.kv_per_tok
        return {"ms": ms, "tok_s": batch * 1000.0 / ms, "mean_ctx": mean_ctx, "marks": (t0, t1),
                "launches": eng.launches_per_decode_step(batch) + 1,  # + the argmax
                "gbs": bytes_step / (ms * 1e-3) / 1e9, "finite": finite}

    def prefill_run(self, tokens, repeats=3):
        """One prompt of `tokens` tokens in one step; the best of `repeats` after a warm-up."""
        import torch

        eng = self.eng
        prompt = torch.randint(0, self.V, (tokens,), generator=self.g).tolist()
        times, finite = [], True
        for i in range(repeats + 1):
            s = eng.open()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            a.record()
            logits = eng.step([(s, prompt, [tokens - 1])])
            b.record()
            torch.cuda.synchronize()
            finite = finite and bool(torch.isfinite(logits).all().item())
            eng.close(s)
            if i >= 1:
                times.append(a.elapsed_time(b))
        eng.check_errors()
        pms = min(times)
        fl = prefill_flops(self.cfg, self.layers, tokens)
        return {"ms": pms, "tok_s": tokens * 1000.0 / pms, "flops": fl, "tflops": fl / (pms * 1e-3) / 1e12,
                "finite": finite}

    def generate_run(self, prompts, new_tokens, sampling=None):
        """Decode tokens a second through the entry point: the time of
        1 + new_tokens tokens a prompt less the time of 1 (the prefill and the
        first pick), host ids in and out."""
        import torch

        m = self.model
        m.generate(prompts, 3, sampling)  # warm: allocations, graphs of the first sizes
        torch.cuda.synchronize()
        ta = time.perf_counter()
        m.generate(prompts, 1, sampling)
        torch.cuda.synchronize()
        tb = time.perf_counter()
        out = m.generate(prompts, 1 + new_tokens, sampling)
        torch.cuda.synchronize()
        tc = time.perf_counter()
        s = (tc - tb) - (tb - ta)
        n = sum(len(o) - 1 for o in out)
        return {"tok_s": n / s, "seconds": s, "tokens": n, "steps": new_tokens}


# ---- a second design beside the closest existing one, at equal sizes (--design) ----
# Layer sizes that resemble a real model's; `kv_rank` stays within what the
# tensor-core attention kernels take (256).  The Qwen3 model beside each has the
# same width, depth, head count, head size, feed-forward width, vocabulary and
# attention span (all layers slide over the same window).
DESIGN_SIZES = {
    "w1024": {"width": 1024, "layers": 8, "heads": 8, "dim": 128, "q_rank": 384, "kv_rank": 128, "window": 1024,
              "m_heads": 4, "m_dim": 128, "m_vdim": 256, "ff": 4096, "experts": 8, "top": 2, "expert_ff": 2048,
              "vocab": 32768},
    "w2048": {"width": 2048, "layers": 8, "heads": 16, "dim": 128, "q_rank": 768, "kv_rank": 256, "window": 1024,
              "m_heads": 8, "m_dim": 128, "m_vdim": 256, "ff": 8192, "experts": 16, "top": 4, "expert_ff": 2048,
              "vocab": 32768},
    "w4096": {"width": 4096, "layers": 4, "heads": 32, "dim": 128, "q_rank": 1536, "kv_rank": 256, "window": 1024,
              "m_heads": 16, "m_dim": 128, "m_vdim": 256, "ff": 12288, "experts": 16, "top": 4, "expert_ff": 3072,
              "vocab": 32768},
}


def kegasun_config(z):
    lat = {"type": "latent_attention",
           "mixer": {"heads": z["heads"], "dim": z["dim"], "vdim": z["dim"], "q_rank": z["q_rank"],
                     "kv_rank": z["kv_rank"], "mask": {"size": z["window"]}, "scale": z["dim"] ** -0.5}}
    rec = {"type": "mlstm", "mixer": {"heads": z["m_heads"], "dim": z["m_dim"], "vdim": z["m_vdim"], "gate_cap": 15.0}}
    dense = {"kind": "dense", "ff": z["ff"]}
    moe = {"kind": "moe", "expert": {"ff": z["expert_ff"]}, "router": {"experts": z["experts"], "top": z["top"]}}
    pattern = [(rec, dense), (lat, moe), (lat, dense), (lat, moe)]
    layers = [dict(pattern[i % 4][0], mlp=pattern[i % 4][1]) for i in range(z["layers"])]
    return {"architecture": "Kegasun", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-5},
            "embedding": {"scale": 1.0, "bigram": {"buckets": 65521, "mul_prev": 127, "mul_cur": 7}},
            "layers": layers}


def pakarax_config(z):
    """Pakarax at the sizes of `z`: every layer an attention (a quarter as many
    key/value heads, filters of four taps) beside a gated linear recurrence of
    the model's width, dense and routed feed-forwards in turn (the routed ones
    with a shared expert); all layers form one pass of the loop, so that the
    number of layer runs and the weights equal the models beside it."""
    pair = {"type": "parallel",
            "mixer": {"left": {"heads": z["heads"], "kv_heads": max(1, z["heads"] // 4), "dim": z["dim"],
                               "vdim": z["dim"], "conv": 4, "scale": z["dim"] ** -0.5,
                               "q_temp": {"coef": 0.3, "every": 128}},
                      "right": {"width": z["width"], "blocks": z["heads"], "conv": 4}}}
    dense = {"kind": "dense", "ff": z["ff"], "limit": 7.0}
    moe = {"kind": "moe", "expert": {"ff": z["expert_ff"], "limit": 7.0},
           "router": {"experts": z["experts"], "top": z["top"]}, "shared": {"ff": z["expert_ff"], "limit": 7.0}}
    layers = [dict(pair, mlp=(dense, moe)[i % 2]) for i in range(z["layers"])]
    return {"architecture": "Pakarax", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-5},
            "logit_scale": 1.0, "logit_softcap": 30.0, "loop": {"start": 0, "stop": z["layers"], "times": 1},
            "layers": layers}


def purusun_config(z):
    """Purusun at the sizes of `z`: attention layers (a quarter as many key/value
    heads, half of each head rotated with scaled frequencies, the window of the
    models beside it with four kept first tokens) and selective-scan layers (twice
    the width as channels, 16 states, a step-size rank of width / 16, four taps) in
    turn, every layer with a squared-ReLU feed-forward, four residual streams."""
    att = {"type": "attention",
           "mixer": {"heads": z["heads"], "kv_heads": max(1, z["heads"] // 4), "dim": z["dim"], "vdim": z["dim"],
                     "scale": z["dim"] ** -0.5,
                     "rot": {"base": 500000.0, "dims": z["dim"] // 2,
                             "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}},
                     "mask": {"size": z["window"], "keep_first": 4}}}
    scan = {"type": "mamba1", "mixer": {"inner": 2 * z["width"], "state": 16, "dt_rank": z["width"] // 16, "conv": 4}}
    dense = {"kind": "dense", "ff": z["ff"]}
    layers = [dict((att, scan)[i % 2], mlp=dense) for i in range(z["layers"])]
    return {"architecture": "Purusun", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-5},
            "streams": 4, "layers": layers}


def zelinex_config(z):
    """Zelinex at the sizes of `z`: layers of a sigmoid-weight attention (a quarter
    as many key/value heads, half of each head rotated, the window of the models
    beside it) beside a state-space recurrence of the model's width (heads of 64
    channels, 128 states, two groups, four taps) with a dense feed-forward, in turn
    with layers of a delta rule of the model's width (heads of 64) with experts and a
    shared expert; all layers form one pass of the loop, so that the number of layer
    runs equals the models beside it."""
    pair = {"type": "parallel",
            "mixer": {"left": {"heads": z["heads"], "kv_heads": max(1, z["heads"] // 4), "dim": z["dim"],
                               "vdim": z["dim"], "scale": z["dim"] ** -0.5,
                               "rot": {"base": 500000.0, "dims": z["dim"] // 2}, "mask": {"size": z["window"]}},
                      "right": {"heads": z["width"] // 64, "vdim": 64, "state": 128, "groups": 2, "conv": 4,
                                "norm_groups": 2},
                      "left_scale": 0.75, "right_scale": 0.55}}
    delta = {"type": "general_delta", "mixer": {"heads": z["width"] // 64, "dim": 64}}
    dense = {"kind": "dense", "ff": z["ff"]}
    moe = {"kind": "moe", "expert": {"ff": z["expert_ff"]},
           "router": {"experts": z["experts"], "top": z["top"], "scale": 1.25}, "shared": {"ff": z["expert_ff"]}}
    layers = [dict((pair, delta)[i % 2], mlp=(dense, moe)[i % 2]) for i in range(z["layers"])]
    return {"architecture": "Zelinex", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-5},
            "residual_mult": 0.8, "loop": {"start": 0, "stop": z["layers"], "times": 1}, "layers": layers}


def zivulix_config(z):
    """Zivulix at the sizes of `z`: of four layers two are a gated delta rule (heads of
    128 keys and values, twice the width of values, half as many query/key heads, four
    taps), one is a capped attention (a quarter as many key/value heads, half of each head
    rotated, the window of the models beside it, mixed values) and one a latent attention
    (a rotated part of 64 beside the models' head size, every earlier key), every layer
    with a feed-forward."""
    delta = {"type": "delta", "mixer": {"heads": z["width"] // 64, "kv_heads": z["width"] // 128, "dim": 128,
                                        "vdim": 128, "conv": 4}}
    att = {"type": "attention",
           "mixer": {"heads": z["heads"], "kv_heads": max(1, z["heads"] // 4), "dim": z["dim"], "vdim": z["dim"],
                     "scale": z["dim"] ** -0.5, "softcap": 50.0, "v_mix": True,
                     "rot": {"base": 500000.0, "dims": z["dim"] // 2, "scaling": {"factor": 4.0}},
                     "mask": {"size": z["window"]}}}
    lat = {"type": "latent_attention",
           "mixer": {"heads": z["heads"], "dim": z["dim"], "rot_dim": 64, "vdim": z["dim"], "kv_rank": z["kv_rank"],
                     "scale": (z["dim"] + 64) ** -0.5, "rot": {"base": 500000.0, "dims": 64}}}
    pattern = [delta, att, delta, lat]
    layers = [dict(pattern[i % 4], mlp={"kind": "dense", "ff": z["ff"]}) for i in range(z["layers"])]
    return {"architecture": "Zivulix", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-5},
            "layers": layers}


def pidodra_config(z):
    """Pidodra at the sizes of `z`: of four layers two are a latent attention (a rotated part
    of 64 beside the models' head size, queries through a latent, a gate per element), one a
    grouped attention (a quarter as many key/value heads, YaRN frequencies, a gate per head)
    and one the same with that one's keys and values, every layer with experts in four groups
    of which two are kept; every earlier key."""
    lat = {"type": "latent_attention",
           "mixer": {"heads": z["heads"], "dim": z["dim"], "rot_dim": 64, "vdim": z["dim"], "q_rank": z["q_rank"],
                     "kv_rank": z["kv_rank"], "scale": (z["dim"] + 64) ** -0.5, "rot": {"base": 500000.0, "dims": 64}}}
    att = {"heads": z["heads"], "kv_heads": max(1, z["heads"] // 4), "dim": z["dim"], "vdim": z["dim"],
           "scale": z["dim"] ** -0.5,
           "rot": {"base": 500000.0, "dims": z["dim"],
                   "scaling": {"factor": 4.0, "original": 8192, "fast": 32.0, "slow": 1.0}}}
    moe = {"kind": "moe", "expert": {"ff": z["expert_ff"]},
           "router": {"experts": z["experts"], "top": z["top"], "scale": 1.5, "groups": {"count": 4, "keep": 2}}}
    layers = []
    for i in range(z["layers"]):
        mixer = [lat, {"type": "attention", "mixer": att}, lat,
                 {"type": "attention", "mixer": dict(att, kv_from=i - 2)}][i % 4]
        layers.append(dict(mixer, mlp=moe))
    return {"architecture": "Pidodra", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-5},
            "embedding": {"scale": 1.0}, "postln_alpha": 2.0, "layers": layers}


def qwen3_config_like(z):
    cfg = dict(QWEN3_8B)
    cfg.update({"num_hidden_layers": z["layers"], "hidden_size": z["width"], "num_attention_heads": z["heads"],
                "num_key_value_heads": max(1, z["heads"] // 4), "head_dim": z["dim"], "intermediate_size": z["ff"],
                "vocab_size": z["vocab"], "use_sliding_window": True, "sliding_window": z["window"],
                "layer_types": ["sliding_attention"] * z["layers"]})
    return cfg


def design_comparison(args) -> int:
    """Prefill and decode throughput of a design (`--design`) beside Qwen3 at
    equal sizes (and, for Pakarax, beside Kegasun too: the model with a
    recurrence and experts; for Zelinex beside Pakarax: the model with two mixers
    side by side, experts and a loop; for Zivulix beside Kegasun, the model with a latent
    attention, and Zelinex, the model with a delta rule; for Pidodra beside Zivulix, the
    model with a rotated latent attention, and Kegasun, the model with a latent attention and
    experts), with every phase's time in a
    prefill and in a decode step."""
    import torch

    from reflex_b200 import ops
    from reflex_b200.api import Model
    from reflex_b200.weights import random_model_on_device

    pk = peaks()
    torch.cuda.set_device(0)
    T, B, P, steps = PREFILL_TOKENS, args.batch, PROMPT, max(16, min(args.steps, 64))
    mine = args.design
    beside = [("qwen3", qwen3_config_like)] + {
        "pakarax": [("kegasun", kegasun_config)], "zelinex": [("pakarax", pakarax_config)],
        "zivulix": [("kegasun", kegasun_config), ("zelinex", zelinex_config)],
        "pidodra": [("zivulix", zivulix_config), ("kegasun", kegasun_config), ("zelinex", zelinex_config)]}.get(mine, [])
    mine_config = {"kegasun": kegasun_config, "pakarax": pakarax_config, "purusun": purusun_config,
                   "zelinex": zelinex_config, "zivulix": zivulix_config, "pidodra": pidodra_config}[mine]
    out = {"metric": f"prefill and decode tokens/s, {mine} beside " + " and ".join(n for n, _ in beside)
                     + " at equal sizes", "unit": "tokens/s",
           "dtype": "bf16", "data": "synthetic: seeded uniform token ids, random-init weights",
           "prefill_tokens": T, "decode_batch": B, "decode_prompt": P, "decode_steps": steps,
           "peaks": {"hbm_gbs": pk["hbm_gbs"], "bf16_tflops": pk["bf16_tflops"], "of": pk["source"]}, "sizes": {}}
    names = [n for n in args.sizes.split(",") if n]
    for name in names:
        z = DESIGN_SIZES[name]
        row = {}
        for design, cfg in [(mine, mine_config(z))] + [(n, f(z)) for n, f in beside]:
            lm = random_model_on_device(cfg, 0, torch.bfloat16, "cuda:0")
            model = Model(lm, max_tokens=B * (P + steps + 128) + T + 256, max_batch=B)
            eng = model.engine
            g = torch.Generator().manual_seed(1)
            V = z["vocab"]
            prompt = torch.randint(0, V, (T,), generator=g).tolist()
            times = []
            for i in range(4):
                s = eng.open()
                a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                torch.cuda.synchronize()
                a.record()
                logits = eng.step([(s, prompt, [T - 1])])
                b.record()
                torch.cuda.synchronize()
                eng.close(s)
                if i:
                    times.append(a.elapsed_time(b))
            finite = bool(torch.isfinite(logits).all().item())
            pms = min(times)
            # decode: B sequences from P-token prompts, ids fed from the device
            prompts = torch.randint(0, V, (B, P), generator=g).tolist()
            seqs = [eng.open() for _ in range(B)]
            logits = eng.step([(s, p, [P - 1]) for s, p in zip(seqs, prompts)])
            ids = [torch.empty((B,), dtype=torch.int32, device="cuda:0") for _ in range(2)]
            scratch = torch.empty((B * 128,), dtype=torch.float32, device="cuda:0")
            ops.argmax(logits, out=ids[0], scratch=scratch)
            for i in range(4):
                logits = eng.step_decode(seqs, ids[i % 2], borrow=True)
                ops.argmax(logits, out=ids[(i + 1) % 2], scratch=scratch)
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            a.record()
            for i in range(4, 4 + steps):
                logits = eng.step_decode(seqs, ids[i % 2], borrow=True)
                ops.argmax(logits, out=ids[(i + 1) % 2], scratch=scratch)
            b.record()
            torch.cuda.synchronize()
            dms = a.elapsed_time(b) / steps
            finite = finite and bool(torch.isfinite(logits).all().item())
            launches = eng.launches_per_decode_step(B)
            # every phase's time: one eager prefill and one eager decode step with events at the marks
            ops.PROFILE = True
            eng.use_graphs = False
            s = eng.open()
            eng.step([(s, prompt, [T - 1])])
            phases_prefill = {k: round(v, 4) for k, v in ops.LAST_PROFILE.items()}
            eng.close(s)
            eng.step([(q, [1], [0]) for q in seqs])
            eng.step([(q, [1], [0]) for q in seqs])
            phases_decode = {k: round(v, 4) for k, v in ops.LAST_PROFILE.items()}
            ops.PROFILE = False
            for q in seqs:
                eng.close(q)
            eng.check_errors()
            weight_bytes = sum(t.untyped_storage().nbytes() for t in _model_tensors(lm))
            row[design] = {"prefill_ms": pms, "prefill_tok_s": T * 1000.0 / pms, "decode_ms": dms,
                           "decode_tok_s": B * 1000.0 / dms, "decode_launches": launches, "finite": finite,
                           "weight_bytes": weight_bytes, "phases_prefill_ms": phases_prefill,
                           "phases_decode_ms": phases_decode}
            del model, eng, lm
            import gc

            gc.collect()
            torch.cuda.empty_cache()
        for other, _ in beside:
            suffix = "" if other == "qwen3" else f"_vs_{other}"
            row["prefill_ratio" + suffix] = row[mine]["prefill_tok_s"] / row[other]["prefill_tok_s"]
            row["decode_ratio" + suffix] = row[mine]["decode_tok_s"] / row[other]["decode_tok_s"]
        out["sizes"][name] = row
    print(json.dumps(out))
    return 0


def _model_tensors(lm):
    """Every weight tensor a model's parts hold (for a count of bytes)."""
    import torch

    seen, out = set(), []

    def walk(o, depth=0):
        if isinstance(o, torch.Tensor):
            # by storage: a part's rows of a stacked matrix are a view, not more weights
            key = o.untyped_storage().data_ptr()
            if o.is_cuda and key not in seen:
                seen.add(key)
                out.append(o)
        elif isinstance(o, (list, tuple)):
            for x in o:
                walk(x, depth + 1)
        elif hasattr(o, "__dict__") and depth < 8:  # a mixer may hold mixers of its own
            for x in vars(o).values():
                walk(x, depth + 1)

    walk(lm)
    return out


def main() -> int:
    global PROMPT, CONTEXT
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=200)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--layers", type=int, default=0, help="fewer layers than the model has (0 = all)")
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--no-points", action="store_true", help="skip the batch 1 / 64 decode points")
    ap.add_argument("--no-prefill", action="store_true", help="skip the 2,048-token prefill")
    ap.add_argument("--shape", default="8b", choices=sorted(SHAPES), help="layer sizes of the headline (default: Qwen3-8B)")
    ap.add_argument("--arms", default="8b,14b,32b",
                    help="workloads beside the headline: 14b and 32b add their points (default: all)")
    ap.add_argument("--prompt", type=int, default=PROMPT, help="prompt tokens before the decode steps")
    ap.add_argument("--context", type=int, default=CONTEXT, help="cache positions per sequence")
    ap.add_argument("--design", default="", choices=["", "kegasun", "pakarax", "pidodra", "purusun", "zelinex", "zivulix"],
                    help="instead of the headline: this design beside Qwen3 at equal sizes (prefill, decode, phases)")
    ap.add_argument("--sizes", default="w1024,w2048,w4096", help="with --design: which of the sizes " +
                    ", ".join(sorted(DESIGN_SIZES)))
    args = ap.parse_args()
    if args.design and args.impl == "ours":
        return design_comparison(args)
    PROMPT = args.prompt
    CONTEXT = max(args.context, args.prompt + max(args.steps, 0 if args.no_points else POINT_STEPS) + args.warmup + 64)

    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable":
                          "lateos-ai/reflex is a Rust crate (no setup.py/pyproject.toml; pip: 'Directory is "
                          "not installable') and no Rust toolchain exists in this image"}))
        return 0
    if args.gpus != 1:
        print(f"bench.py measures one GPU only: --gpus {args.gpus} is not supported (this library is single-GPU)")
        return 2
    if args.warmup < 3:
        args.warmup = 3
    arms = [a for a in args.arms.split(",") if a]
    for a in arms:
        if a not in SHAPES:
            print(f"--arms: unknown workload {a!r}; known: {sorted(SHAPES)}")
            return 2

    import torch

    from reflex_b200.engine.batch import layout
    from reflex_b200.sampling import SamplingParams

    pk = peaks()
    torch.cuda.set_device(0)
    max_batch = max(args.batch, 1 if args.no_points else 64)
    arm = Arm(args.shape, args.layers, max_batch * CONTEXT, max_batch)
    cfg, layers = arm.cfg, arm.layers

    sampler = ClockSampler()
    sampler.start()
    time.sleep(0.3)
    head = arm.decode_run(args.batch, PROMPT, args.steps, args.warmup, sampler)
    clocks = sampler.summary(*head["marks"])
    finite = head["finite"]

    # end to end through the Python entry point: host ids in, host ids out
    prompts = torch.randint(0, arm.V, (args.batch, PROMPT), generator=arm.g).tolist()
    n_e2e = min(args.steps, 128)
    gen = arm.generate_run(prompts, n_e2e)
    _, words = layout(args.batch, args.batch, args.batch)
    e2e = {"value": gen["tok_s"], "unit": "tokens/s", "steps": n_e2e,
           "h2d_bytes_per_step": words * 4, "d2h_bytes_per_step": args.batch * 4}

    out = {
        "metric": f"decode tokens/s at batch {args.batch} (Qwen3-{args.shape.upper()} bf16, {PROMPT}-token prompts, "
                  f"context {CONTEXT})",
        "value": head["tok_s"], "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
        "ms_per_step": head["ms"], "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic: seeded uniform token ids, random-init weights N(0, 0.02)",
        "impl": "ours",
        "config": {
            "model": f"Qwen3-{args.shape.upper()} layer sizes", "layers": layers, "layers_full_model": arm.full_layers,
            "hidden_size": cfg["hidden_size"], "intermediate_size": cfg["intermediate_size"],
            "num_attention_heads": cfg["num_attention_heads"],
            "num_key_value_heads": cfg["num_key_value_heads"], "head_dim": cfg["head_dim"],
            "vocab_size": arm.V, "global_batch": args.batch, "seq_len": CONTEXT, "prompt_tokens": PROMPT,
            "mean_context": head["mean_ctx"], "parallelism": "single GPU", "cache_page_tokens": 64,
            "l2": "inputs larger than L2 (15 GB of weights per step), no flush",
            "peaks": pk["source"], "points_steps": POINT_STEPS, "arms": ",".join(arms),
        },
        "clocks": clocks, "e2e": e2e, "gpu_launches": head["launches"] * args.steps,
        "roofline": {"bound": "hbm", "achieved": head["gbs"], "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": head["gbs"] / pk["hbm_gbs"], "of": pk["source"]},
    }

    if not args.no_prefill:
        p = arm.prefill_run(PREFILL_TOKENS)
        finite = finite and p["finite"]
        out["prefill"] = {"value": p["tok_s"], "tokens": PREFILL_TOKENS, "ms": p["ms"],
                          "frac": p["tflops"] / pk["bf16_tflops"], "flops": p["flops"],
                          "peak_tflops": pk["bf16_tflops"], "of": pk["source"]}
    points, fracs = {}, {}
    if not args.no_points:
        for b in (1, 64):
            r = arm.decode_run(b, PROMPT, POINT_STEPS, 4)
            finite = finite and r["finite"]
            points[f"decode_b{b}"] = r["tok_s"]
            fracs[f"decode_b{b}"] = r["gbs"] / pk["hbm_gbs"]
        points[f"decode_b{args.batch}"] = head["tok_s"]
        fracs[f"decode_b{args.batch}"] = head["gbs"] / pk["hbm_gbs"]
    arm.free()
    del arm

    if not args.no_points:
        try:
            if "14b" in arms and args.shape == "8b":
                # 16 prompts of seeded lengths in [64, 2048], 128 steps at temperature 0.7, context 4,096
                a14 = Arm("14b", 0, 16 * 4096, 16)
                lens = torch.randint(64, 2049, (16,), generator=torch.Generator().manual_seed(14)).tolist()
                ps = [torch.randint(0, a14.V, (n,), generator=a14.g).tolist() for n in lens]
                r = a14.generate_run(ps, 128, SamplingParams(temperature=0.7, seed=14))
                ctx_sum = sum(n + 1 + 64.5 for n in lens)
                gbs = (a14.weight_bytes + ctx_sum * a14.kv_per_tok) / (r["seconds"] / r["steps"]) / 1e9
                points["qwen3_14b_b16_unequal_t0.7_decode"] = r["tok_s"]
                fracs["qwen3_14b_b16_unequal_t0.7_decode"] = gbs / pk["hbm_gbs"]
                a14.free()
                del a14
            if "32b" in arms and args.shape == "8b":
                # batch 32 from 1,024-token prompts over 256 steps; one 8,192-token prefill; 8,192 a slot
                a32 = Arm("32b", 0, 32 * 8192, 32)
                r = a32.decode_run(32, 1024, POINT_STEPS, 4)
                p = a32.prefill_run(8192, repeats=2)
                finite = finite and r["finite"] and p["finite"]
                points["qwen3_32b_b32_decode"] = r["tok_s"]
                fracs["qwen3_32b_b32_decode"] = r["gbs"] / pk["hbm_gbs"]
                points["qwen3_32b_prefill_8192"] = p["tok_s"]
                fracs["qwen3_32b_prefill_8192"] = p["tflops"] / pk["bf16_tflops"]
                a32.free()
                del a32
        except Exception as e:  # the headline stands; the point that failed says why
            points["error"] = f"{type(e).__name__}: {e}"[:300]
        out["points"] = points
        out["points_frac"] = fracs
    out["finite"] = finite
    sampler.stop()
    print(json.dumps(out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
