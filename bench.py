#!/usr/bin/env python3
"""Decode and prefill throughput of the engine on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference]

Default workload: the layer sizes of BASELINE.json's configs[2] (Llama-2-7B sizes with one kv
head: 32 layers, width 4096, 32 heads of 128, SwiGLU 11008, vocabulary 32000), random bfloat16
weights, batch 8, context 4096.  A step is one decode step of the whole batch.  One JSON line
is printed: ``value`` = decoded tokens per second timed on the device over exactly K steps;
``e2e`` = the same through ``Engine.step()`` with host tokens in and out; ``prefill`` = one
2,048-token prompt; ``roofline`` = bytes a decode step must read / time / measured HBM peak;
``points`` = decode at batch 1 and 64.
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

FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}


def load_json(name):
    try:
        with open(os.path.join(ROOT, name)) as f:
            return json.load(f)
    except (OSError, ValueError):
        return None


def peaks():
    m = load_json("MEASURED_PEAKS.json") or {}
    out, src = dict(FALLBACK_PEAKS), "fallback"
    def find(d, key):
        if isinstance(d, dict):
            if key in d and isinstance(d[key], (int, float)):
                return float(d[key])
            for v in d.values():
                r = find(v, key)
                if r is not None:
                    return r
        return None
    for k in ("hbm_gbs", "bf16_tflops"):
        v = find(m, k)
        if v:
            out[k], src = v, "measured"
    out["source"] = src
    return out


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while the timed region runs."""
    Q = ("clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
         "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.rows, self.proc = [], None

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", "0", f"--query-gpu={self.Q}", "--format=csv,noheader,nounits",
                                          "-lms", "100"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.rows.append([c.strip() for c in line.split(",")])

    def stop(self):
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        time.sleep(0.15)
        self.proc.terminate()
        sm = [float(r[0]) for r in self.rows if r and r[0].replace(".", "").isdigit()]
        mx = [float(r[1]) for r in self.rows if len(r) > 1 and r[1].replace(".", "").isdigit()]
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = [n for i, n in enumerate(names) if any(len(r) > 3 + i and r[3 + i].lower().startswith("active") for r in self.rows)]
        return {"sm_mhz": statistics.median(sm) if sm else None, "sm_max_mhz": max(mx) if mx else None,
                "reasons": reasons, "samples": len(sm)}


def model_numbers(cfg, layers):
    """Bytes a decode step must read and flops of a prefill, from the shapes (2 bytes per value)."""
    d, F, V, Hq, Hkv = cfg["d_model"], cfg["hidden_size"], cfg["vocab_size"], cfg["num_heads"], cfg["num_kv_heads"]
    D = d // Hq
    per_layer = (Hq + 2 * Hkv) * D * d + d * Hq * D + 3 * F * d + 2 * d
    weights = layers * per_layer + V * d + d                     # lm_head + final norm; embedding rows are counted per token
    kv_per_token = layers * 2 * Hkv * D * 2
    return {"matmul_params": layers * ((Hq + 2 * Hkv) * D * d + d * Hq * D + 3 * F * d), "weights_bytes": 2 * weights,
            "kv_bytes_per_token": kv_per_token, "head_dim": D, "lm_head_params": V * d}


def build_engine(cfg, layers, batch, ctx, graphs, seed=0):
    import torch
    from tiny_transformer_inference_engine_b200 import Engine, ModelConfig, EngineConfig, CacheConfig, SchedulerConfig
    from tiny_transformer_inference_engine_b200.weights import random_tensors
    mc = ModelConfig.from_dict({**cfg, "num_layers": layers})
    w = random_tensors(mc, seed, store_dtype="bfloat16", device="cuda:0")
    page = 64
    pages = batch * (-(-ctx // page)) + 2 * batch + 2        # admission keeps a growth page per running request
    ec = EngineConfig(dtype="bfloat16", device="cuda:0", use_cuda_graphs=True,
                      cache=CacheConfig(block_size=page, num_gpu_blocks=pages),
                      sched=SchedulerConfig(max_num_seqs=batch, max_num_batched_tokens=max(2048, batch),
                                            cudagraph_batch_sizes=graphs))
    eng = Engine(mc, w, ec)
    del w
    torch.cuda.empty_cache()
    return eng


def timed(fn, steps):
    import torch
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    a.record()
    for i in range(steps):
        fn(i)
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b)


def decode_kernel_path(eng, batch, start_len, steps, warmup, vocab, synthetic_fill, prefix="b"):
    """Device-timed decode: K steps of (metadata copy, captured model step, sampling kernel)."""
    import torch
    from tiny_transformer_inference_engine_b200 import StepEntry, SamplingParams
    mgr, g = eng.manager, torch.Generator().manual_seed(1)
    rids = [f"{prefix}{i}" for i in range(batch)]
    for rid in rids:
        mgr.admit(rid)
        eng.sampler.set_request(mgr.slot_of[rid], SamplingParams(temperature=0.8, seed=mgr.slot_of[rid]))
    if synthetic_fill:
        for rid in rids:
            mgr.extend(rid, 0, start_len)
        for grp in mgr.groups:
            grp.kv.normal_(0, 0.5)
    else:
        chunk = 2048
        for rid in rids:
            for s in range(0, start_len, chunk):
                n = min(chunk, start_len - s)
                mgr.extend(rid, s, s + n)
                eng.stepper.step([StepEntry(rid, s, torch.randint(0, vocab, (n,), generator=g).tolist(), [])])
    tokens = torch.randint(0, vocab, (warmup + steps, batch), generator=g).tolist()
    slot_ids = torch.tensor([mgr.slot_of[r] for r in rids], dtype=torch.int32, device="cuda:0")
    pos = [start_len]

    def one(i, base=0):
        for rid in rids:
            mgr.extend(rid, pos[0], pos[0] + 1)
        entries = [StepEntry(rid, pos[0], [tokens[base + i][j]], [0]) for j, rid in enumerate(rids)]
        logits = eng.stepper.step(entries, eng.sampler)         # a captured step samples inside its graph
        if eng.stepper.last_tokens is None:
            eng.sampler.sample(logits, slot_ids)
        pos[0] += 1

    for i in range(warmup):
        one(i)
    l0 = eng.ops.launches
    ms = timed(lambda i: one(i, warmup), steps)
    for rid in rids:
        mgr.release(rid)
    return ms, pos[0], eng.ops.launches - l0


WORKLOADS = {
    # Falcon-7B widths in Llama style, a mixed batch of 32 requests
    "falcon_mixed": dict(
        cfg=dict(architecture="mqa_gpt", vocab_size=65024, d_model=4544, num_layers=32, num_heads=71, num_kv_heads=1,
                 hidden_size=18176, max_seq_len=2048, rope_theta=10000.0, rms_norm_eps=1e-5, bias=False, dtype="bfloat16"),
        requests=32, prompt_lo=64, prompt_hi=1024, new_tokens=128, token_budget=2048, page=64),
    # Gemma-2B layer sizes, 6,144-token prompts in 512-token portions beside decode
    "gemma_chunked": dict(
        cfg=dict(architecture="mqa_gpt", vocab_size=256000, d_model=2048, num_layers=18, num_heads=8, num_kv_heads=1,
                 hidden_size=16384, max_seq_len=8192, rope_theta=10000.0, rms_norm_eps=1e-6, bias=False, dtype="bfloat16"),
        requests=16, prompt_lo=6144, prompt_hi=6144, new_tokens=256, token_budget=512, page=64),
}


def run_workload(name, pk, layers=None, split_classes=True):
    """One of BASELINE.json's serving workloads through ``Engine.generate`` (host token lists in and out): requests are
    admitted, their prompts cut into portions under the token budget and run beside the decoded tokens of the others.
    Timed by the host's clock around the whole call, after one untimed run of the same workload; the faster of two timed
    runs counts.  ``frac`` is the sum
    over the steps of the time each would need at the roofline (the larger of bytes / HBM peak and flops / bf16 peak)
    divided by the time taken."""
    import torch
    from tiny_transformer_inference_engine_b200 import Engine, ModelConfig, EngineConfig, CacheConfig, SchedulerConfig, SamplingParams
    from tiny_transformer_inference_engine_b200.weights import random_tensors
    w = WORKLOADS[name]
    cfg, n_req, page = w["cfg"], w["requests"], w["page"]
    full_layers = cfg["num_layers"]
    layers = layers or full_layers
    mc = ModelConfig.from_dict({**cfg, "num_layers": layers})
    g = torch.Generator().manual_seed(3)
    lens = torch.randint(w["prompt_lo"], w["prompt_hi"] + 1, (n_req,), generator=g).tolist()
    prompts = [torch.randint(0, cfg["vocab_size"], (n,), generator=g).tolist() for n in lens]
    pages = sum(-(-(n + w["new_tokens"]) // page) for n in lens) + 2 * n_req + 2
    ec = EngineConfig(dtype="bfloat16", device="cuda:0", use_cuda_graphs=True, split_step_classes=split_classes,
                      cache=CacheConfig(block_size=page, num_gpu_blocks=pages),
                      sched=SchedulerConfig(max_num_seqs=n_req, max_num_batched_tokens=w["token_budget"],
                                            cudagraph_batch_sizes=[1, 2, 4, 8, 16, 32]))
    eng = Engine(mc, random_tensors(mc, 0, store_dtype="bfloat16", device="cuda:0"), ec)
    torch.cuda.empty_cache()
    nums = model_numbers(cfg, layers)
    params = SamplingParams(max_new_tokens=w["new_tokens"], temperature=0.8, ignore_eos=True)
    log = []
    inner = eng.stepper.step

    def logged(entries, *a, **k):                                  # what each step ran, for the roofline sum
        log.append([(e.start, len(e.tokens)) for e in entries])
        return inner(entries, *a, **k)

    eng.stepper.step = logged
    eng.generate(prompts, params)                                   # untimed: graphs captured, kernels loaded
    # timed twice, the faster run counts: the host's clock around a whole workload also sees whatever else the host does
    # (the same workload on an idle and on a busy host of this pool: 1.22 and 1.3-2.3 s with the GPU's clocks unchanged)
    secs = []
    for _ in range(2):
        log.clear()
        l0 = eng.ops.launches
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        out = eng.generate(prompts, params)
        torch.cuda.synchronize()
        secs.append(time.perf_counter() - t0)
        assert all(len(o) == w["new_tokens"] for o in out)
    sec = min(secs)
    ideal, mixed_steps = 0.0, 0
    Hq, D = cfg["num_heads"], nums["head_dim"]
    for step in log:
        T = sum(n for _, n in step)
        keys = sum(s + n for s, n in step)
        flops = 2 * T * nums["matmul_params"] + 2 * len(step) * nums["lm_head_params"] \
            + layers * 4 * Hq * D * sum(n * s + n * (n + 1) // 2 for s, n in step)
        bytes_ = nums["weights_bytes"] + keys * nums["kv_bytes_per_token"]
        ideal += max(bytes_ / (pk["hbm_gbs"] * 1e9), flops / (pk["bf16_tflops"] * 1e12))
        mixed_steps += any(n == 1 for _, n in step) and any(n > 1 for _, n in step)
    gen = n_req * w["new_tokens"]
    res = {"value": gen / sec, "unit": "generated tokens/s", "seconds": sec, "seconds_of_both_runs": [round(t, 4) for t in secs], "prompt_tokens": sum(lens), "generated_tokens": gen,
           "all_tokens_per_s": (sum(lens) + gen) / sec, "steps": len(log), "mixed_steps": int(mixed_steps),
           "roofline_frac": ideal / sec, "layers": layers, "layers_in_config": full_layers,
           "requests": n_req, "token_budget": w["token_budget"], "page_size": page, "gpu_launches": eng.ops.launches - l0,
           "preemptions": eng.stats()["preemptions"]}
    del eng
    torch.cuda.empty_cache()
    return res


# ------------------------------------------------------------------------------------------ --design munevik
def munevik_config(width, heads, layers=4):
    """A Munevik model at layer sizes that resemble a real model's: latent attention with a 256-value cache row, a
    recurrent block as wide as the model in blocks of 128, a clamped GLU of 4 x width, and 16 experts of width / 2 (two
    chosen, from the best two of four groups) beside a shared expert.  Layer order: attention + dense, recurrent + experts,
    recurrent + experts, attention over the first layer's cache + experts, repeated."""
    att = {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 192, "mask": {"size": 1024},
           "rot": {"base": 10000.0, "dims": 64}, "scale": 192 ** -0.5}
    rec = {"width": width, "blocks": width // 128, "conv": 4}
    moe = {"kind": "moe", "expert": {"ff": width // 2}, "shared": {"ff": width},
           "router": {"experts": 16, "top": 2, "groups": {"count": 4, "keep": 2}, "scale": 1.0}}
    dense = {"kind": "dense", "ff": 4 * width, "limit": 7.0}
    out = []
    for i in range(layers):
        k = i % 4
        if k == 0:
            out.append({"type": "latent_attention", "mixer": dict(att), "mlp": dense})
        elif k == 3:
            out.append({"type": "latent_attention", "mixer": dict(att, kv_from=i - 3), "mlp": moe})
        else:
            out.append({"type": "rglru", "mixer": dict(rec), "mlp": moe})
    return {"architecture": "Munevik", "vocab": 32000, "width": width, "postln_alpha": 1.0, "norm": {"eps": 1e-6}, "layers": out,
            "max_seq_len": 4096}


def mizupel_config(width, heads, layers=4):
    """A Mizupel model at layer sizes that resemble a real model's: grouped-query attention with heads of 128 (eight query heads
    per kv head), four convolution taps, 64 rotated values, a window of 1,024 keys and soft-capped scores; a matrix memory of
    width / 128 heads with 64 key and 128 value channels; time mixing with heads of 64 and a decay path of rank 64; feed-forwards
    of 4 x width.  Layer order: attention + feed-forward, matrix memory, time mixing + feed-forward, attention + feed-forward,
    repeated."""
    att = {"heads": heads, "kv_heads": max(1, heads // 8), "dim": 128, "vdim": 128, "conv": 4, "mask": {"size": 1024},
           "rot": {"base": 10000.0, "dims": 64, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}},
           "scale": 128 ** -0.5, "softcap": 50.0}
    mem = {"heads": heads, "dim": 64, "vdim": 128, "gate_cap": 15.0}
    mix = {"heads": width // 64, "dim": 64, "decay_rank": 64}
    ff = {"kind": "dense", "ff": 4 * width}
    out = []
    for i in range(layers):
        k = i % 4
        if k in (0, 3):
            out.append({"type": "attention", "mixer": dict(att), "mlp": ff})
        elif k == 1:
            out.append({"type": "mlstm", "mixer": dict(mem), "mlp": None})
        else:
            out.append({"type": "wkv", "mixer": dict(mix), "mlp": ff})
    return {"architecture": "Mizupel", "vocab": 32000, "width": width, "norm": {"eps": 1e-6}, "logit_softcap": 30.0, "layers": out,
            "max_seq_len": 4096}


def mokalorn_config(width, heads, layers=4):
    """A Mokalorn model at layer sizes that resemble a real model's: grouped-query attention with heads of 128 (eight query heads
    per kv head), the keys as values, 64 rotated values and chunks of 1,024 positions; a second attention with a value projection,
    one kv head per eight heads and a query temperature; retention with width / 128 heads of 128 key and 128 value channels;
    feed-forwards of 16 experts of width / 2 and two identity experts, four chosen.  Layer order: chunked attention, retention,
    causal attention, retention, repeated."""
    rot = {"base": 10000.0, "dims": 64}
    att = {"heads": heads, "kv_heads": max(1, heads // 8), "dim": 128, "vdim": 128, "mask": {"size": 1024}, "rot": rot, "scale": 128 ** -0.5}
    att2 = {"heads": heads, "kv_heads": max(1, heads // 8), "dim": 128, "vdim": 128, "q_temp": {"coef": 0.1, "every": 512}, "scale": 128 ** -0.5}
    ret = {"heads": heads, "dim": 128, "vdim": 128, "rot": {"base": 10000.0, "dims": 128},
           "decay": [1.0 - 2.0 ** (-5 - 3 * i / max(1, heads - 1)) for i in range(heads)]}
    moe = {"kind": "moe", "expert": {"ff": width // 2, "limit": 7.0}, "router": {"experts": 16, "identity": 2, "top": 4}}
    out = []
    for i in range(layers):
        k = i % 4
        if k == 0:
            out.append({"type": "attention", "mixer": dict(att), "mlp": moe})
        elif k == 2:
            out.append({"type": "attention_2", "mixer": dict(att2), "mlp": moe})
        else:
            out.append({"type": "retention", "mixer": dict(ret), "mlp": moe})
    return {"architecture": "Mokalorn", "vocab": 32000, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
            "logit_softcap": 30.0, "layers": out, "max_seq_len": 4096}


def dabilorn_config(width, heads, layers=4):
    """A Dabilorn model at layer sizes that resemble a real model's: latent attention with heads of 128 + 64 rotated values, a
    256-value cache row (latent of 192), a query latent of 3/8 of the width and YaRN-rescaled frequencies; grouped-query attention
    with sigmoid weights, heads of 128 (eight query heads per kv head), 64 rotated values and chunks of 1,024 positions; time
    mixing with heads of 64 and a decay path of rank 64; four convolution taps in front of every mixer; feed-forwards of 16
    experts of width / 2, four chosen, beside a gated shared expert of the model's width.  Layer order: time mixing, latent
    attention, sigmoid attention, latent attention, repeated."""
    lat = {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 192, "q_rank": 3 * width // 8, "scale": 192 ** -0.5,
           "rot": {"base": 10000.0, "dims": 64, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    att = {"heads": heads, "kv_heads": max(1, heads // 8), "dim": 128, "vdim": 128, "mask": {"size": 1024},
           "rot": {"base": 10000.0, "dims": 64}, "scale": 128 ** -0.5}
    mix = {"heads": width // 64, "dim": 64, "decay_rank": 64}
    moe = {"kind": "moe", "expert": {"ff": width // 2}, "router": {"experts": 16, "top": 4}, "shared": {"ff": width}}
    kinds = (("wkv", mix), ("latent_attention", lat), ("attention", att), ("latent_attention", lat))
    out = [{"type": kinds[i % 4][0], "mixer": dict(kinds[i % 4][1]), "mlp": moe} for i in range(layers)]
    return {"architecture": "Dabilorn", "vocab": 32000, "width": width, "norm": {"eps": 1e-6}, "canon": {"taps": 4}, "layers": out,
            "max_seq_len": 4096}


def renanex_config(width, heads, layers=4):
    """A Renanex model at layer sizes that resemble a real model's: selective scan with twice the width as channels, 16 states, a
    step-size rank of width / 16 and four convolution taps; linear attention with width / 128 heads of 128 key and 128 value
    channels; attention with scores mixed over the heads, heads of 128 (eight query heads per kv head), YaRN-rescaled
    rotation, a window of 1,024 keys that keeps the first four, and blended values; feed-forwards of 4 x width.  Layer order:
    selective scan, linear attention, attention, attention, repeated."""
    ssm = {"inner": 2 * width, "state": 16, "dt_rank": width // 16, "conv": 4}
    lin = {"heads": heads, "dim": 128, "vdim": 128, "decay": [1.0 - 2.0 ** (-5 - 3 * i / max(1, heads - 1)) for i in range(heads)]}
    att = {"heads": heads, "kv_heads": max(1, heads // 8), "dim": 128, "vdim": 128, "mask": {"size": 1024, "keep_first": 4},
           "rot": {"base": 10000.0, "dims": 128, "scaling": {"factor": 4.0, "original": 2048, "fast": 32.0, "slow": 1.0}},
           "scale": 128 ** -0.5, "v_mix": True}
    ff = {"kind": "dense", "ff": 4 * width}
    kinds = (("mamba1", ssm), ("lightning", lin), ("attention", att), ("attention", att))
    out = [{"type": kinds[i % 4][0], "mixer": dict(kinds[i % 4][1]), "mlp": ff} for i in range(layers)]
    return {"architecture": "Renanex", "vocab": 32000, "width": width, "norm": {"eps": 1e-6}, "logit_scale": 1.0, "logit_softcap": 30.0,
            "layers": out, "max_seq_len": 4096}


def fokurax_config(width, heads, layers=4):
    """A Fokurax model at layer sizes that resemble a real model's: grouped-query attention with heads of 128 (eight query heads per
    kv head), 64 rotated values with YaRN-rescaled frequencies, chunks of 1,024 positions; a gelu-gated feed-forward of 4 x width in
    every fourth layer, 16 experts of width / 2, four per token, in the others; 256 side values per layer and token.  Layer
    order: attention + dense, attention + experts, two layers on the second one's cache with experts, repeated."""
    att = {"heads": heads, "kv_heads": max(1, heads // 8), "dim": 128, "vdim": 128, "mask": {"size": 1024}, "scale": 128 ** -0.5,
           "rot": {"base": 10000.0, "dims": 64, "scaling": {"factor": 4.0, "original": 2048, "fast": 32.0, "slow": 1.0}}}
    moe = {"kind": "moe", "expert": {"ff": width // 2}, "router": {"experts": 16, "top": 4}}
    out = []
    for i in range(layers):
        k = i % 4
        out.append({"type": "attention", "mixer": dict(att, kv_from=i - k + 1) if k >= 2 else dict(att),
                    "mlp": {"kind": "dense", "ff": 4 * width} if k == 0 else moe})
    return {"architecture": "Fokurax", "vocab": 32000, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0}, "residual_mult": 0.7,
            "logit_softcap": 30.0, "token_side": {"dim": 256}, "layers": out, "max_seq_len": 4096}


DESIGNS = {"munevik": ("Munevik", munevik_config, 1024), "mizupel": ("Mizupel", mizupel_config, 1024),
           "mokalorn": ("Mokalorn", mokalorn_config, 0), "dabilorn": ("Dabilorn", dabilorn_config, 0),
           "renanex": ("Renanex", renanex_config, 1024), "fokurax": ("Fokurax", fokurax_config, 0)}     # name, configuration, window


def like_config(width, heads, layers=4):
    """The closest existing model at equal size: pre-norm multi-query attention blocks with heads of 128 and SwiGLU of 4 x width."""
    return dict(architecture="mqa_gpt", vocab_size=32000, d_model=width, num_layers=layers, num_heads=width // 128, num_kv_heads=1,
                hidden_size=4 * width, max_seq_len=4096, rope_theta=10000.0, rms_norm_eps=1e-6, bias=False, dtype="bfloat16")


class OpRecorder:
    """Wraps the kernel library's operations: notes every call of one step (name, arguments), so that each can be timed alone
    afterwards, and its algorithmic bytes and flops from the shapes."""
    NAMES = ("embed", "add_rmsnorm", "rmsnorm_rows", "linear", "linear_swiglu", "rope_table", "rope_store", "paged_attention",
             "scale_add_layernorm", "cast_rows", "latent_store", "latent_query", "gate_heads", "batched_linear", "causal_conv",
             "rglru_scan", "glu", "linear_glu", "grouped_glu", "moe_route", "moe_plan", "grouped_linear", "moe_combine",
             "qkv_conv_rope_store", "conv_tail_update", "gate_head_rows", "token_shift_mix", "wkv_scan", "mlstm_scan", "head_norm_gate",
             "activation", "linear_act", "wkv_decay", "mlstm_gates", "rotate_heads", "retention_scan", "stream_conv", "proj_row_rms",
             "rmsnorm_cols", "grouped_act", "sandwich_norm", "joint_qkv_store", "paged_attention_joint", "selective_scan", "activation_rows", "linear_narrow",
             "residual_sum", "token_gate", "moe_plan_table")

    def __init__(self, ops):
        self.ops, self.calls, self.orig, self.depth = ops, [], {}, 0

    def __enter__(self):
        for n in self.NAMES:
            fn = getattr(self.ops, n)
            self.orig[n] = fn
            setattr(self.ops, n, self._wrap(n, fn))
        return self

    def __exit__(self, *a):
        for n, fn in self.orig.items():
            setattr(self.ops, n, fn)

    def _wrap(self, name, fn):
        def call(*args, **kw):
            self.depth += 1                                      # (an operation made of others is noted whole, not its parts)
            try:
                out = fn(*args, **kw)
            finally:
                self.depth -= 1
            if self.depth == 0:
                self.calls.append((name, fn, args, kw, out))
            return out
        return call


def _tensor_bytes(x):
    import torch
    if isinstance(x, torch.Tensor):
        return x.numel() * x.element_size()
    if isinstance(x, (list, tuple)):
        return sum(_tensor_bytes(v) for v in x)
    if isinstance(x, dict):
        return sum(_tensor_bytes(v) for v in x.values())
    return 0


def op_cost(name, args, kw, out, kv_lens, window):
    """(bytes that must move, flops) of one recorded call, from its shapes."""
    import torch
    flops = 0
    if name in ("wkv_scan", "mlstm_scan"):
        # the step's rows in and out, each request's state row read and written once; the recurrence's arithmetic is 32-bit on
        # the ordinary cores: three (wkv) or four (mlstm) multiply-adds per state element and token, returned as a second count
        if name == "wkv_scan":
            r, state, n, H, D = args[0], args[5], args[10], args[11], args[12]
            T, per_tok, fma = r.shape[0], 3 * H * D * r.element_size() + 8 * H * D, 3 * H * D * D
        else:
            q, state, n, H, D, Dv = args[0], args[4], args[9], args[10], args[11], args[12]
            T, per_tok, fma = q.shape[0], (2 * H * D + H * Dv) * q.element_size() + 4 * H * Dv + 8 * H, 4 * H * D * Dv
        row = state[0].numel() * 4
        return T * per_tok + 2 * n * row, ("fp32", 2 * T * fma)
    if name == "retention_scan":                                   # like the other matrix-state scans: two multiply-adds per state element and token
        q, v, state, n, H, D, Dv = args[0], args[2], args[4], args[7], args[8], args[9], args[10]
        T = q.shape[0]
        return T * (2 * H * D * 4 + H * Dv * v.element_size() + 4 * H * Dv) + 2 * n * state[0].numel() * 4, ("fp32", 2 * T * 2 * H * D * Dv)
    if name == "selective_scan":                                   # (u, dt, ..., A, D, bc, ..., z, state, ..., requests, states): three multiply-adds per state and token and an
                                                                    # exponential, of which an SM does 16 a clock: it takes the time of eight multiply-adds
        u, bc, z, S, n, N = args[0], args[5], args[8], args[9], args[15], args[16]
        T, I = u.shape
        return T * (3 * I * u.element_size() + 4 * I + bc.shape[1] * bc.element_size()) + 2 * n * I * N * 4, ("fp32", 2 * T * 8 * I * N)
    if name == "sandwich_norm":                                    # (resid, delta, ...): the stream read and written (gathered rows: read), the delta read, one row out
        rows = kw.get("num_rows") or args[0].shape[0]
        per = args[0].shape[1] * ((4 if kw.get("rows") is not None else 8) + args[6].element_size())
        return rows * per + _tensor_bytes(args[1]) * rows // args[0].shape[0], 0
    if name == "residual_sum":                                     # (resid, a, f): the stream read and written, every term read, the copy written
        ex = kw.get("experts")
        return 2 * _tensor_bytes(args[0]) + _tensor_bytes(list(args[1:3])) + _tensor_bytes([ex[0], ex[1]["pos_of_pair"]] if ex else []) + _tensor_bytes(out), 0
    if name == "token_gate":                                       # (z, ids, table, col0, n, ...): of the table one layer's values per token
        return _tensor_bytes([args[0], args[1], out]) + args[1].shape[0] * args[4] * args[2].element_size(), 0
    if name == "moe_plan_table":                                   # (tables, ids, ...): a row of every layer's table per token
        return args[1].shape[0] * (1 + args[0].shape[0] * args[0].shape[2]) * 4 + _tensor_bytes(out), 0
    if name == "activation_rows":                                  # (x, cols, ...)
        return args[0].shape[0] * args[1] * args[0].element_size() + _tensor_bytes(out), 0
    if name == "joint_qkv_store":                                  # the projected row read, joint query rows written, joint key and value rows stored
        T, H, W = args[0].shape[0], args[1], args[5]
        used = H * args[3] + args[2] * (args[3] + args[4])
        es = args[0].element_size()
        return T * es * (used + 2 * W) + _tensor_bytes(out), ("fp32", 2 * T * H * H * args[3])
    if name == "paged_attention_joint":                            # plain grouped attention's bytes and products, and the mixing of the scores (H x H per key)
        q, H, G, W, Dv, kp = args[0], args[1], args[2], args[3], args[4], args[5]
        D, keep = W // G, kw.get("keep_first") or 0
        seen = sum(sum(min(p + 1, (window or p + 1) + keep) for p in range(L - n, L)) for L, n in kv_lens)
        vis = sum(min(L, (window + n + keep) if window else L) for L, n in kv_lens)
        return (q.shape[0] * H * (D + Dv) + vis * G * (D + Dv)) * q.element_size(), seen * H * (2 * D + 2 * Dv + 2 * H)
    if name == "rotate_heads":                                     # (src, heads, dim, ...): the rotated columns read, 32-bit rows written
        return args[0].shape[0] * args[1] * args[2] * args[0].element_size() + _tensor_bytes(out), 0
    if name == "qkv_conv_rope_store":                              # pages and state rows are pools: count the rows read and written
        return 2 * _tensor_bytes(args[0]) + _tensor_bytes(out), 0
    if name == "conv_tail_update":                                 # (proj, channels, taps, tail, qsl, slots, requests)
        return 2 * args[6] * (args[2] - 1) * args[1] * 4, 0
    if name == "token_shift_mix":
        return _tensor_bytes([args[0], out]), 0
    if name in ("wkv_decay", "mlstm_gates"):
        return _tensor_bytes([args[0], out]), 0
    if name in ("head_norm_gate", "gate_head_rows"):
        return _tensor_bytes([args[0], args[1], out]), 0
    if name in ("linear", "linear_swiglu", "linear_glu", "linear_act", "linear_narrow"):
        x, w = args[0], args[1]
        flops = 2 * x.shape[0] * w.shape[0] * w.shape[1]
        return _tensor_bytes([x, w, out]), flops
    if name == "batched_linear":
        x, w = args[0], args[1]
        return _tensor_bytes([w, out]) + x.numel() * x.element_size(), 2 * x.shape[0] * x.shape[1] * w.shape[1] * w.shape[2]
    if name == "stream_conv":                                      # (resid, weights, ...): the stream's rows read, the mixer's input written
        return _tensor_bytes([args[0], out]), 0
    if name == "proj_row_rms":                                     # (proj, nq, nk, eps): the q and k columns read
        return args[0].shape[0] * (args[1] + args[2]) * args[0].element_size() + _tensor_bytes(out), 0
    if name == "rmsnorm_cols":                                     # (proj, col0, width, ...)
        return args[0].shape[0] * args[2] * args[0].element_size() + _tensor_bytes(out), 0
    if name in ("grouped_linear", "grouped_glu", "grouped_act"):
        x, w, plan = args[0], args[1], args[2]
        rows = plan["pairs"]
        return _tensor_bytes([w, out]) + rows * w.shape[2] * x.element_size(), 2 * rows * w.shape[1] * w.shape[2]
    if name == "paged_attention":
        q, H, Hkv, D, kp, vp = args[0], args[1], args[2], args[3], args[4], args[5]
        planes = 1 if kp.data_ptr() == vp.data_ptr() else 2
        chunk = kw.get("chunk") or 0
        if chunk:                                                   # a token sees the keys of its own chunk up to itself
            seen = [[p % chunk + 1 for p in range(L - n, L)] for L, n in kv_lens]
            vis = [min(L, n + (L - n) % chunk) for L, n in kv_lens]
            fl = sum(4 * H * D * sum(s) for s in seen)
        else:
            vis = [min(L, window + n) if window else L for L, n in kv_lens]
            fl = sum(4 * H * D * n * (min(L, window) if window else (L - n / 2)) for L, n in kv_lens)
        kv_bytes = sum(vis) * Hkv * D * kp.element_size() * planes
        return 2 * q.shape[0] * H * D * q.element_size() + kv_bytes, fl
    if name in ("rope_store", "latent_store"):
        x = args[0]
        return 2 * x.shape[-2] * x.shape[-1] * x.element_size() if name == "rope_store" else _tensor_bytes(x) // 4, 0
    if name == "embed":
        return 2 * _tensor_bytes(args[2]), 0
    tensors = [a for a in list(args) + list(kw.values())]
    skip = 0
    if name in ("causal_conv", "rglru_scan"):                   # the state tensor holds every slot: count the step's rows only
        skip = 0
    return _tensor_bytes(tensors) + _tensor_bytes(out) - skip, 0


FP32_NOMINAL_FLOPS = 148 * 128 * 2 * 1.965e9        # 148 SMs x 128 lanes x one multiply-add per clock at the highest SM clock (nominal, not measured)


def time_ops(eng, entries_fn, pk, kv_lens, window, iters=8):
    """Runs one step with every operation recorded, then times each recorded call alone (a replayed graph of ``iters`` calls);
    returns rows (operation, calls, microseconds, fraction of its roofline)."""
    import torch
    with OpRecorder(eng.ops) as rec:
        entries_fn()
        torch.cuda.synchronize()
    rows = {}
    for name, fn, args, kw, out in rec.calls:
        try:
            us = eng.ops._graph_time(lambda: fn(*args, **kw), iters) * 1e3 / iters
        except Exception:                                        # (an operation that cannot be captured alone is timed plainly)
            torch.cuda.synchronize()
            us = timed(lambda i: fn(*args, **kw), iters) * 1e3 / iters
        b, f = op_cost(name, args, kw, out, kv_lens, window)
        if isinstance(f, tuple):                                  # 32-bit arithmetic on the ordinary cores: against their nominal rate
            ideal = max(b / (pk["hbm_gbs"] * 1e9), f[1] / FP32_NOMINAL_FLOPS) * 1e6
        else:
            ideal = max(b / (pk["hbm_gbs"] * 1e9), f / (pk["bf16_tflops"] * 1e12)) * 1e6
        key = name
        if name in ("linear", "batched_linear", "grouped_linear", "linear_swiglu", "linear_glu", "grouped_glu", "linear_act", "grouped_act", "linear_narrow"):
            w = args[1]
            key = f"{name} {list(w.shape)}"
        r = rows.setdefault(key, {"calls": 0, "us": 0.0, "ideal_us": 0.0})
        r["calls"] += 1; r["us"] += us; r["ideal_us"] += ideal
    for r in rows.values():
        r["frac"] = round(r["ideal_us"] / r["us"], 3) if r["us"] else None
        r["us"], r["ideal_us"] = round(r["us"], 1), round(r["ideal_us"], 2)
    return rows


def run_design(args, pk):
    """Prefill and decode throughput of a design (``--design``) at a few sizes, beside the closest existing model (``--beside``:
    the multi-query GPT, or another design) at equal width and depth, with every operation of a step timed alone against its
    roofline."""
    import torch
    from tiny_transformer_inference_engine_b200 import Engine, ModelConfig, EngineConfig, CacheConfig, SchedulerConfig, StepEntry, SamplingParams
    from tiny_transformer_inference_engine_b200.weights import random_tensors
    sizes = [(1024, 8), (2048, 16), (4096, 32)] if not args.sizes else [(int(w), int(w) // 128) for w in args.sizes.split(",")]
    Tp, batch, ctx, K, W = 2048, args.batch, 2048, args.steps, max(args.warmup, 3)
    report = {}
    for width, heads in sizes:
        design_name, design_config, design_window = DESIGNS[args.design]
        beside = args.beside or "mqa_gpt"
        beside_cfg = (DESIGNS[beside][1] if beside in DESIGNS else like_config)(width, heads, args.layers or 4)
        for label, cfg in ((args.design, design_config(width, heads, args.layers or 4)), (beside, beside_cfg)):
            mc = ModelConfig.from_dict(cfg)
            page = 64
            pages = batch * (ctx // page + 4) + Tp // page + 8
            # (the prompt's step is replayed from a graph like the decode steps: a step of a hundred launches at these sizes is
            # otherwise timed by the host's launches, not by the GPU)
            ec = EngineConfig(dtype="bfloat16", device="cuda:0", use_cuda_graphs=True, step_graph_max_tokens=Tp,
                              cache=CacheConfig(block_size=page, num_gpu_blocks=pages),
                              sched=SchedulerConfig(max_num_seqs=batch + 1, max_num_batched_tokens=4096, cudagraph_batch_sizes=[batch]))
            eng = Engine(mc, random_tensors(mc, 0, store_dtype="bfloat16", device="cuda:0"), ec)
            vocab = mc.vocab_size
            g = torch.Generator().manual_seed(0)
            ptoks = torch.randint(0, vocab, (Tp,), generator=g).tolist()

            def prefill_once(_=None):
                eng.manager.admit("p")
                eng.manager.extend("p", 0, Tp)
                eng.stepper.step([StepEntry("p", 0, ptoks, [Tp - 1])])
                eng.manager.release("p")

            for _ in range(3):
                prefill_once()
            p_ms = timed(prefill_once, 5) / 5
            window = DESIGNS[label][2] if label in DESIGNS else 0
            saved_cap, eng.stepper.capture_repeated = eng.stepper.capture_repeated, False     # the recorded step runs eagerly
            p_ops = time_ops(eng, prefill_once, pk, [(Tp, Tp)], window)
            eng.stepper.capture_repeated = saved_cap
            ms, end_len, launches = decode_kernel_path(eng, batch, ctx - (W + K), K, W, vocab, synthetic_fill=False)
            # one decode step, eagerly, for the per-operation times
            rids = [f"d{i}" for i in range(batch)]
            for rid in rids:
                eng.manager.admit(rid)
                eng.manager.extend(rid, 0, ctx)
            for grp in eng.manager.groups:
                grp.kv.normal_(0, 0.5)
            saved, eng.stepper.graph_batch_sizes = eng.stepper.graph_batch_sizes, []

            def decode_once():
                eng.stepper.step([StepEntry(rid, ctx - 1, [7 + 11 * i], [0]) for i, rid in enumerate(rids)])     # (different tokens: experts may go by the id)

            d_ops = time_ops(eng, decode_once, pk, [(ctx, 1)] * batch, window)
            eng.stepper.graph_batch_sizes = saved
            for rid in rids:
                eng.manager.release(rid)
            report[f"{label}_{width}"] = {
                "prefill_tokens_per_s": round(Tp / (p_ms / 1e3)), "prefill_ms": round(p_ms, 3),
                "decode_tokens_per_s": round(batch * K / (ms / 1e3)), "decode_ms_per_step": round(ms / K, 4),
                "decode_launches_per_step": launches // K, "layers": len(mc.layers) if label in DESIGNS else mc.num_layers,
                "prefill_ops": p_ops, "decode_ops": d_ops}
            del eng
            torch.cuda.empty_cache()
    print(json.dumps({"design": DESIGNS[args.design][0], "beside": args.beside or "mqa_gpt", "dtype": "bf16", "data": "synthetic token ids, random-init weights",
                      "prefill_tokens": Tp, "decode_batch": batch, "decode_context": ctx, "steps": K, "warmup": W,
                      "peaks": pk, "sizes": report}))
    return 0


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--design", default=None, choices=("munevik", "mizupel", "mokalorn", "dabilorn", "renanex", "fokurax"), help="prefill and decode of this design at a few sizes beside the closest existing model, with per-operation times")
    ap.add_argument("--beside", default=None, choices=("mqa_gpt", "munevik", "mizupel", "mokalorn", "dabilorn", "renanex", "fokurax"), help="with --design: the model it is timed beside (default: the multi-query GPT)")
    ap.add_argument("--sizes", default=None, help="with --design: comma-separated model widths (multiples of 128)")
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=("ours", "reference"))
    ap.add_argument("--layers", type=int, default=None, help="fewer layers than the configuration (named in config)")
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--no-points", action="store_true")
    ap.add_argument("--no-workloads", action="store_true", help="skip the Falcon-width and Gemma-size serving workloads")
    ap.add_argument("--only-workload", default=None, choices=sorted(WORKLOADS), help="run one serving workload and print its record")
    ap.add_argument("--no-class-split", action="store_true", help="with --only-workload: mixed steps as one attention launch (the comparison)")
    args = ap.parse_args()

    if args.impl == "reference":
        # The unmodified reference from baseline/_ref, in a process of its own (none of this package is imported there):
        # baseline/reference_arm.py builds its PagedTransformer at the same sizes and times its generate_batched loop.
        if args.gpus != 1:
            print(json.dumps({"impl": "reference", "unavailable": "the reference runs on one GPU"}))
            return 0
        cmd = [sys.executable, os.path.join(ROOT, "baseline", "reference_arm.py"), "--steps", str(args.steps),
               "--warmup", str(max(args.warmup, 3)), "--batch", str(args.batch)]
        if args.layers:
            cmd += ["--layers", str(args.layers)]
        try:
            run = subprocess.run(cmd, capture_output=True, text=True, timeout=1500)
            lines = [l for l in run.stdout.strip().split("\n") if l.startswith("{")]
            if run.returncode == 0 and lines:
                print(lines[-1])
            else:
                tail = " ".join((run.stderr or run.stdout).split())[-300:]
                print(json.dumps({"impl": "reference", "unavailable": f"the reference's process ended with code {run.returncode}: {tail}"}))
        except subprocess.TimeoutExpired:
            print(json.dumps({"impl": "reference", "unavailable": "the reference's process did not finish in 1500 s"}))
        return 0
    if args.gpus != 1:
        print(f"this engine runs on one GPU; --gpus {args.gpus} is not supported")
        return 2
    if args.warmup < 3:
        args.warmup = 3

    import torch
    if args.design:
        return run_design(args, peaks())
    if args.only_workload:
        print(json.dumps({args.only_workload: run_workload(args.only_workload, peaks(), args.layers, not args.no_class_split)}))
        return 0
    cfg = dict(architecture="mqa_gpt", vocab_size=32000, d_model=4096, num_layers=32, num_heads=32, num_kv_heads=1,
               hidden_size=11008, max_seq_len=4096, rope_theta=10000.0, rms_norm_eps=1e-5, bias=False, dtype="bfloat16")
    full_layers = cfg["num_layers"]
    layers = args.layers or full_layers
    ctx, batch, K, W = cfg["max_seq_len"], args.batch, args.steps, args.warmup
    pk = peaks()
    nums = model_numbers(cfg, layers)

    eng = build_engine(cfg, layers, max(batch, 1), ctx, sorted({1, batch}))
    vocab = cfg["vocab_size"]

    # ---- prefill of 2,048 tokens (one request, empty cache)
    from tiny_transformer_inference_engine_b200 import StepEntry, SamplingParams
    g = torch.Generator().manual_seed(0)
    Tp = 2048
    ptoks = torch.randint(0, vocab, (Tp,), generator=g).tolist()

    def prefill_once(_):
        eng.manager.admit("p")
        eng.manager.extend("p", 0, Tp)
        eng.stepper.step([StepEntry("p", 0, ptoks, [Tp - 1])])
        eng.manager.release("p")

    for i in range(3):
        prefill_once(i)
    p_ms = timed(prefill_once, 3) / 3
    p_flops = 2 * Tp * nums["matmul_params"] + 4 * cfg["num_heads"] * nums["head_dim"] * (Tp * (Tp + 1) // 2) * layers \
        + 2 * nums["lm_head_params"]
    prefill = {"value": Tp / (p_ms / 1e3), "tokens": Tp, "ms": p_ms,
               "frac": p_flops / (p_ms / 1e3) / (pk["bf16_tflops"] * 1e12)}

    # ---- decode, device-timed
    start_len = ctx - (W + K)
    clocks = ClockSampler(); clocks.start()
    ms, end_len, launches = decode_kernel_path(eng, batch, start_len, K, W, vocab, synthetic_fill=False)
    clock_rec = clocks.stop()
    ms_per_step = ms / K
    value = batch * K / (ms / 1e3)
    mean_ctx = (start_len + W + end_len) / 2
    step_bytes = nums["weights_bytes"] + batch * cfg["d_model"] * 2 + batch * mean_ctx * nums["kv_bytes_per_token"]
    achieved = step_bytes / (ms_per_step / 1e3) / 1e9
    roofline = {"bound": "hbm", "achieved": achieved, "peak": pk["hbm_gbs"], "unit": "GB/s", "frac": achieved / pk["hbm_gbs"],
                "of": pk["source"]}

    # ---- decode end to end through Engine.step(): host tokens in, host tokens out
    # requests that finish their prompt early decode while the others still prefill, so each gets
    # room for those extra tokens and none finishes inside the timed region
    prefill_steps = -(-batch * start_len // 2048) + batch
    room = W + K + prefill_steps + 2
    e2e_prompt = ctx - room
    prompts = torch.randint(0, vocab, (batch, e2e_prompt), generator=g).tolist()
    for p in prompts:
        eng.add_request(p, SamplingParams(max_new_tokens=room, temperature=0.8, ignore_eos=True))
    while any(r.remaining > 1 for r in list(eng.scheduler.running) + list(eng.scheduler.waiting)) or eng.scheduler.waiting:
        eng.step()
    for _ in range(W):
        eng.step()
    n_e2e = K
    got = [0]

    def e2e_step(_):
        got[0] += len(eng.step())

    e_ms = timed(e2e_step, n_e2e)
    assert got[0] == batch * n_e2e, (got[0], batch, n_e2e)
    for r in list(eng.scheduler.running):
        eng.manager.release(r.rid)
    eng.scheduler.running.clear()
    h2d = 4 * (8 * (batch + 4) + batch * (-(-ctx // 64)) + 64)          # the step's packed int32 metadata
    e2e = {"value": got[0] / (e_ms / 1e3), "unit": "tokens/s", "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": 4 * batch,
           "steps": n_e2e}

    # ---- other batch sizes
    points = {}
    eng = None
    torch.cuda.empty_cache()
    if not args.no_points:
        for b in (1, 64):
            e2 = build_engine(cfg, layers, b, ctx, [b])
            k2 = min(K, 32)
            # twice on the same engine, the better one kept: these are side figures of a few dozen steps, and one slow
            # stretch of the GPU (seen once: 9 x) would otherwise stand as the figure
            m2 = min(decode_kernel_path(e2, b, ctx - (W + k2), k2, W, vocab, synthetic_fill=True, prefix=tag)[0] for tag in ("p", "q"))
            points[f"decode_b{b}"] = b * k2 / (m2 / 1e3)
            del e2
            torch.cuda.empty_cache()

    workloads = {}
    if not args.no_workloads:
        for name in WORKLOADS:
            workloads[name] = run_workload(name, pk)

    out = {
        "metric": "decode tokens/s (batch 8, context 4096)", "value": value, "unit": "tokens/s", "n_gpus": 1, "steps": K,
        "warmup": W, "ms_per_step": ms_per_step, "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic token ids, random-init weights",
        "config": {"model": "llama2-7b-sizes-mqa", "global_batch": batch, "seq_len": ctx, "parallelism": "single-gpu",
                   "layers": layers, "layers_in_config": full_layers, "d_model": cfg["d_model"], "heads": cfg["num_heads"],
                   "kv_heads": cfg["num_kv_heads"], "head_dim": nums["head_dim"], "ffn_hidden": cfg["hidden_size"],
                   "vocab": vocab, "page_size": 64, "prompt_len": start_len, "l2": "inputs larger than L2 (weights 11 GB per step)",
                   "cuda_graph": True, "sampling": "temperature 0.8 on device"},
        "e2e": e2e, "gpu_launches": launches, "e2e_prompt_len": e2e_prompt, "prefill": prefill, "roofline": roofline, "points": points, "workloads": workloads, "clocks": clock_rec,
        "impl": "ours",
    }
    print(json.dumps(out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
