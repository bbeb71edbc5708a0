"""Measurement: decode tokens per second of a Llama-4-Scout-shaped model with
random bfloat16 weights on one B200, plus prefill of 2,048 tokens, the decode
step's HBM roofline fraction, and decoding at batch 1 and 64.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference]

A "step" is one decode step of the whole batch.  Prints one JSON line.

Two further workloads print a line of the same kind (they are extra modes; the default line stays the one above):

    python bench.py --config maverick    # Llama-4-Maverick layer shapes, 4 layers (dense, MoE of 128 experts, dense, MoE):
                                         # 64 requests with prompts of 16 to 4,096 tokens through the scheduler
    python bench.py --config long        # Scout layer shapes, 8 layers: a prompt of 131,072 tokens in portions of
                                         # 8,192, then 256 decode steps at batch 1 and at batch 4
    python bench.py --config mibezen     # the Mibezen design beside Llama 4 at equal layer sizes, measured the same way
    python bench.py --config paposun     # the Paposun design beside a dense Llama 4 at equal layer sizes, measured the same way
    python bench.py --config zuzadra     # the Zuzadra design beside Paposun at equal layer sizes, measured the same way
    python bench.py --config fozutar     # the Fozutar design beside Gapevik at equal layer sizes, measured the same way
    python bench.py --config gapevik     # the Gapevik design beside Llama 4 at equal layer sizes, measured the same way
    python bench.py --config sezazen     # the Sezazen design beside Llama 4 at equal layer sizes (three sizes): prefill
                                         # of 2,048 tokens and decode at batch 1 and 8, each with its roofline fraction
"""
from __future__ import annotations

import argparse
import json
import os
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

# Llama-4-Scout layer shapes, 16 layers (the benchmark configuration)
SCOUT = dict(
    architectures=["Llama4ForCausalLM"], num_hidden_layers=16, hidden_size=5120, num_attention_heads=40,
    num_key_value_heads=8, head_dim=128, interleave_moe_layer_step=1, num_local_experts=16,
    num_experts_per_tok=1, intermediate_size=8192, intermediate_size_mlp=16384, vocab_size=202048,
    tie_word_embeddings=False, rope_theta=500000.0,
    rope_scaling=dict(rope_type="llama3", factor=16.0, low_freq_factor=1.0, high_freq_factor=1.0,
                      original_max_position_embeddings=8192),
    attention_chunk_size=8192, no_rope_layer_interval=4, use_qk_norm=True, attn_temperature_tuning=True,
    floor_scale=8192, attn_scale=0.1, rms_norm_eps=1e-5, max_position_embeddings=131072)
FULL_LAYERS = 16
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0}


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    out, src = dict(FALLBACK_PEAKS), "fallback"
    if os.path.isfile(path):
        try:
            raw = json.load(open(path))
            for k in out:
                if isinstance(raw.get(k), (int, float)) and raw[k] > 0:
                    out[k] = float(raw[k])
            src = "measured"
        except (OSError, ValueError):
            pass
    return out, src


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while the timed region runs."""
    Q = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
         "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.rows, self.proc = [], None

    def __enter__(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", "0", f"--query-gpu={self.Q}",
                                          "--format=csv,noheader,nounits", "-lms", "50"],
                                         stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._pump, daemon=True).start()
        except OSError:
            self.proc = None
        return self

    def _pump(self):
        for line in self.proc.stdout:
            self.rows.append([c.strip() for c in line.split(",")])

    def __exit__(self, *exc):
        if self.proc:
            time.sleep(0.25)
            self.proc.terminate()

    def summary(self):
        mhz = sorted(int(r[0]) for r in self.rows if r and r[0].isdigit())
        mx = [int(r[1]) for r in self.rows if len(r) > 1 and r[1].isdigit()]
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = [n for i, n in enumerate(names) if any(len(r) > 2 + i and r[2 + i] == "Active" for r in self.rows)]
        return {"sm_mhz": mhz[len(mhz) // 2] if mhz else None, "sm_max_mhz": max(mx) if mx else None,
                "reasons": reasons, "samples": len(mhz)}


def decode_bytes(model, engine, contexts, distinct_experts):
    """Bytes a decode step has to read: every weight it uses once and the cache of the
    live requests (each layer reads the keys and values its window lets it see)."""
    from spite_b200.parts.feedforward import MoESigmoidPrescaled
    es = 2
    p = model.plan
    total = p.vocab_size * p.hidden_size * es                       # output head (embedding rows are negligible)
    for i, blk in enumerate(model.blocks):
        total += blk.mixer.weight_bytes() + blk.mixer_norm.weight_bytes() + blk.ffn_norm.weight_bytes()
        if isinstance(blk.ffn, MoESigmoidPrescaled):
            total += blk.ffn.active_weight_bytes(distinct_experts[i])
        else:
            total += blk.ffn.weight_bytes()
        win = blk.mixer.window
        for ctx in contexts:
            seen = ctx - win.lowest_visible(ctx - 1)
            total += seen * 2 * blk.mixer.nkv * blk.mixer.hd * es
    return total


def prefill_flops(cfg, T):
    d, hd, nq, nkv = cfg["hidden_size"], cfg["head_dim"], cfg["num_attention_heads"], cfg["num_key_value_heads"]
    f = cfg["intermediate_size"]
    per_layer = 2 * T * d * (nq + 2 * nkv) * hd + 2 * T * nq * hd * d        # projections
    per_layer += 2 * T * d * cfg["num_local_experts"]                          # router
    per_layer += 2 * (2 * T * d * 3 * f)                                       # routed + shared expert
    per_layer += 2 * 2 * nq * hd * T * (T + 1) // 2                            # causal attention
    return cfg["num_hidden_layers"] * per_layer + 2 * d * cfg["vocab_size"]    # one logits row


def prefill_roofline_ms(cfg, T, pk):
    """The time a prefill of T tokens cannot beat kernel by kernel: every product at the sustained bf16 rate or
    the time to read its weights once, whichever is longer, the attention at the bf16 rate, the head's weights."""
    d, hd, nq, nkv = cfg["hidden_size"], cfg["head_dim"], cfg["num_attention_heads"], cfg["num_key_value_heads"]
    f, E, k = cfg["intermediate_size"], cfg["num_local_experts"], cfg["num_experts_per_tok"]
    fl, bw = pk["bf16_tflops_sustained"] * 1e12, pk["hbm_gbs"] * 1e9
    both = lambda flops, nbytes: max(flops / fl, nbytes / bw)
    step = int(cfg.get("interleave_moe_layer_step", 1))
    total = 0.0
    for L in range(cfg["num_hidden_layers"]):
        total += both(2 * T * d * (nq + 2 * nkv) * hd, 2 * d * (nq + 2 * nkv) * hd) + both(2 * T * nq * hd * d, 2 * nq * hd * d)
        total += (2 * 2 * nq * hd * T * (T + 1) // 2) / fl
        if step > 0 and (L + 1) % step == 0:
            total += both(2 * T * d * 3 * f, 2 * 3 * d * f)                             # shared expert
            total += both(2 * T * k * d * 3 * f, 2 * 3 * d * f * min(E, T * k))         # routed experts
        else:
            fm = cfg["intermediate_size_mlp"]
            total += both(2 * T * d * 3 * fm, 2 * 3 * d * fm)
    return (total + 2 * d * cfg["vocab_size"] / bw) * 1e3


def build_model(cfgd):
    import torch
    from spite_b200.config import Llama4Config
    from spite_b200.engine import Model
    from spite_b200.kernels import build as kb
    torch.cuda.set_device(0)
    cfg = Llama4Config.from_dict(cfgd)
    model = Model.from_config(cfg, dtype="bfloat16", device="cuda:0")
    kb.ensure_built(model.kernel_libraries() + ["sampling"])
    model.init_random(seed=0, std=0.02)
    return cfg, model


def distinct_experts(model):
    """Per layer, how many experts the tokens of the last step used (0 for layers without experts)."""
    import torch
    out = []
    for blk in model.blocks:
        r = getattr(blk.ffn, "last_routing", None)
        out.append(torch.unique(r.expert_ids).numel() if r is not None else 0)
    return out


def base_line(metric, value, unit, steps, warmup, ms_per_step, config, data="synthetic (random token ids, random weights N(0,0.02))"):
    return {"metric": metric, "value": round(value, 2), "unit": unit, "n_gpus": 1, "steps": steps, "warmup": warmup,
            "ms_per_step": round(ms_per_step, 4), "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
            "dtype": "bf16", "data": data, "config": config}


def run_maverick(args):
    """sparse routing over 128 experts in mixed batches.  64 requests with prompts of 16
    to 4,096 random tokens and 32 new tokens each go through the public entry point (scheduler, portions of
    prompts beside decoded tokens under a budget of 4,096 tokens a step).  `value` is all tokens run (prompt and
    new) per second of device time; a "step" here is one step of the scheduler."""
    import random
    import torch
    from spite_b200.api import LLM
    cfgd = dict(SCOUT, num_hidden_layers=4, interleave_moe_layer_step=2, num_local_experts=128,
                intermediate_size_mlp=16384, rope_scaling=None)
    cfg, model = build_model(cfgd)
    n_req, new = 64, 32
    llm = LLM(model, ctx=8192, cache_tokens=n_req * 4224, max_requests=n_req, max_batch_tokens=4096)
    rng = random.Random(0)
    prompts = [[rng.randrange(cfg.vocab_size) for _ in range(rng.randint(16, 4096))] for _ in range(n_req)]
    llm.generate(prompts, max_tokens=new, temperature=0.0)            # the same run once untimed: every kernel, shape and graph is warm
    pinned = [torch.tensor(p, dtype=torch.int32).pin_memory() for p in prompts]
    clocks = ClockSampler()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    l0 = model.kernels.launches
    with clocks:
        e0.record()
        outs = llm.generate([p.tolist() for p in pinned], max_tokens=new, temperature=0.0)
        e1.record()
        torch.cuda.synchronize()
    llm.engine.check()
    ms = e0.elapsed_time(e1)
    n_in, n_out = sum(map(len, prompts)), sum(map(len, outs))
    c = llm.last_counters
    line = base_line("tokens/s through the scheduler (Llama-4-Maverick-shaped, 64 requests, prompts 16-4096)",
                     (n_in + n_out) * 1e3 / ms, "tok/s", c["steps"], 1, ms / max(c["steps"], 1),
                     {"model": "llama4-maverick-shaped", "layers": 4, "layers_full": 48, "dense_layers": 2, "moe_layers": 2,
                      "hidden": 5120, "q_heads": 40, "kv_heads": 8, "head_dim": 128, "experts": 128, "top_k": 1,
                      "expert_ffn": 8192, "dense_ffn": 16384, "vocab": 202048, "requests": n_req,
                      "prompt_tokens": n_in, "new_tokens": n_out, "max_batch_tokens": 4096, "page_size": 64,
                      "parallelism": "single-gpu"})
    line.update({"gpu_launches": model.kernels.launches - l0, "clocks": clocks.summary(),
                 "scheduler": {"steps": c["steps"], "preemptions": c["preemptions"], "steps_ahead": c["steps_ahead"]},
                 "e2e": {"value": round((n_in + n_out) * 1e3 / ms, 2), "unit": "tok/s",
                         "h2d_bytes_per_step": round(4 * 4 * (n_in + n_out) / max(c["steps"], 1)), "d2h_bytes_per_step": 4 * n_req,
                         "note": "the whole run goes through LLM.generate: host token lists in, host token lists out"}})
    print(json.dumps(line))


def run_long(args):
    """one request with a prompt of 131,072 tokens run in portions of 8,192 (many chunk
    windows on the chunked layers, the whole context on the layers without rotation), then 256 decode steps at
    batch 1, and the same at batch 4 (four such requests).  `value` is the decode rate at batch 1."""
    import torch
    from spite_b200.engine import Engine, StepEntry
    layers, C, portion, n_dec = args.layers if args.layers != FULL_LAYERS else 8, 131072, 8192, 256
    cfgd = dict(SCOUT, num_hidden_layers=layers, max_position_embeddings=C + 1024)
    cfg, model = build_model(cfgd)
    ks, pk = model.kernels, peaks()
    pk, pk_src = pk
    engine = Engine(model, cache_tokens=4 * (C + 1024), page_size=64, max_requests=4, max_positions=C + 1024)
    g = torch.Generator().manual_seed(3)
    toks = torch.randint(0, cfg.vocab_size, (C,), generator=g, dtype=torch.int32).pin_memory()
    clocks = ClockSampler()

    def prefill(rid):
        ms = []
        for i in range(0, C, portion):
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            engine.step([StepEntry(rid, toks[i:i + portion].tolist(), [portion - 1] if i + portion == C else [])])
            e1.record()
            torch.cuda.synchronize()
            ms.append(e0.elapsed_time(e1))
        return ms

    def decode(rids, steps, warmup=3):
        ids = torch.randint(0, cfg.vocab_size, (steps + warmup, len(rids)), generator=g).tolist()
        for i in range(warmup):
            ks.argmax(engine.step([StepEntry(r, [ids[i][j]], [0]) for j, r in enumerate(rids)]))
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for i in range(warmup, warmup + steps):
            ks.argmax(engine.step([StepEntry(r, [ids[i][j]], [0]) for j, r in enumerate(rids)]))
        e1.record()
        torch.cuda.synchronize()
        ms = e0.elapsed_time(e1) / steps
        ctxs = [engine.cached_tokens(r) for r in rids]
        nbytes = decode_bytes(model, engine, ctxs, [float(n) for n in distinct_experts(model)])
        return ms, nbytes / (ms * 1e-3) / 1e9

    l0 = ks.launches
    with clocks:
        pre = prefill(0)
        ms1, gbs1 = decode([0], n_dec)
    for r in (1, 2, 3):
        prefill(r)
    ms4, gbs4 = decode([0, 1, 2, 3], n_dec)
    engine.check()
    line = base_line("decode tok/s at batch 1 after a 131,072-token prompt (Llama-4-Scout-shaped)", 1e3 / ms1, "tok/s",
                     n_dec, 3, ms1,
                     {"model": "llama4-scout-shaped", "layers": layers, "layers_full": 48, "hidden": 5120, "q_heads": 40,
                      "kv_heads": 8, "head_dim": 128, "experts": 16, "top_k": 1, "expert_ffn": 8192, "vocab": 202048,
                      "chunk": 8192, "nope_every": 4, "global_batch": 1, "seq_len": C, "portion": portion,
                      "page_size": 64, "parallelism": "single-gpu",
                      "l2": "inputs larger than L2 (weights and cache read per step exceed 126 MB)"})
    line.update({
        "gpu_launches": ks.launches - l0, "clocks": clocks.summary(),
        "prefill": {"value": round(C * 1e3 / sum(pre), 1), "tokens": C, "ms": round(sum(pre), 1),
                    "ms_first_portion": round(pre[0], 2), "ms_last_portion": round(pre[-1], 2)},
        "roofline": {"bound": "hbm", "achieved": round(gbs1, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(gbs1 / pk["hbm_gbs"], 4), "peaks": pk_src},
        "points": {"decode_b1": round(1e3 / ms1, 1), "decode_b1_ms": round(ms1, 3), "decode_b1_hbm_frac": round(gbs1 / pk["hbm_gbs"], 4),
                   "decode_b4": round(4e3 / ms4, 1), "decode_b4_ms": round(ms4, 3), "decode_b4_hbm_frac": round(gbs4 / pk["hbm_gbs"], 4)},
        "e2e": {"value": round(1e3 / ms1, 2), "unit": "tok/s", "h2d_bytes_per_step": 4 * (6 + 2 * ((C + 1024) // 64 + 1)),
                "d2h_bytes_per_step": 0, "note": "token ids come from pinned host memory every step; the sampled ids stay on the device"}})
    print(json.dumps(line))


# Layer sizes for the comparison of designs: (name, width, query heads, kv heads, key size, value size, experts,
# experts a token, expert width, shared width, dense width, vocabulary)
DESIGN_SIZES = [
    ("small", 2048, 16, 4, 128, 128, 32, 2, 1024, 2048, 8192, 32768),
    ("medium", 4096, 32, 8, 128, 128, 16, 2, 2048, 4096, 14336, 65536),
    ("medium, value heads of 96", 4096, 32, 8, 128, 96, 16, 2, 2048, 4096, 14336, 65536),
]


def design_configs(size, runs=8):
    """A Sezazen model (one dense layer, a loop of two mixture-of-experts layers run three times, one more such
    layer: eight layer runs) and a Llama 4 model of eight layers with the same widths, heads and experts."""
    name, d, nq, nkv, kd, vd, E, top, f, fs, fd, V = size
    mixer = {"heads": nq, "kv_heads": nkv, "dim": kd, "vdim": vd, "scale": kd ** -0.5}
    moe = {"kind": "moe", "expert": {"ff": f}, "router": {"experts": E, "top": top}, "shared": {"ff": fs}}
    sez = {"architecture": "Sezazen", "vocab": V, "width": d, "max_positions": 8192, "norm": {"eps": 1e-5},
           "embedding": {"scale": 1.0}, "loop": {"start": 1, "stop": 3, "times": 3},
           "layers": [{"type": "attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": fd}}] +
                     [{"type": "attention", "mixer": mixer, "mlp": moe} for _ in range(3)]}
    llama = dict(SCOUT, num_hidden_layers=runs, hidden_size=d, num_attention_heads=nq, num_key_value_heads=nkv,
                 head_dim=kd, num_local_experts=E, num_experts_per_tok=top, intermediate_size=f,
                 intermediate_size_mlp=fd, moe_layers=list(range(1, runs)), vocab_size=V, tie_word_embeddings=True,
                 max_position_embeddings=8192)
    return sez, llama


def mibezen_configs(size, runs=8):
    """A Mibezen model of eight layers (attention with a dense feed-forward, three latent-attention layers with
    experts, attention with experts that blends the first layer's values in, three more latent layers) and a Llama 4
    model of eight layers with the same width, experts and vocabulary, whose attention has the heads of Mibezen's
    attention layers.  A latent row is kv_rank + rot_dim = 128 elements, the largest the tensor-core attention
    kernels take; a chunk is longer than the measured contexts, so every earlier key is read."""
    name, d, nq, nkv, kd, vd, E, top, f, fs, fd, V = size
    att = lambda mix: {"heads": nq, "kv_heads": nkv, "dim": kd, "vdim": kd, "scale": kd ** -0.5, "mask": {"size": 8192}, "v_mix": mix}
    lat = {"heads": 16, "dim": 64, "rot_dim": 32, "vdim": 64, "q_rank": d // 4, "kv_rank": 96, "scale": 96 ** -0.5,
           "rot": {"base": 10000.0, "dims": 32, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    moe = {"kind": "moe", "expert": {"ff": f}, "router": {"experts": E, "top": top}}
    L = lambda t, m, mlp: {"type": t, "mixer": m, "mlp": mlp}
    mib = {"architecture": "Mibezen", "vocab": V, "width": d, "max_positions": 8192, "norm": {"eps": 1e-5}, "logit_softcap": 30.0,
           "layers": [L("attention", att(True), {"kind": "dense", "ff": fd})] + [L("latent_attention", lat, moe)] * 3 +
                     [L("attention", att(True), moe)] + [L("latent_attention", lat, moe)] * 3}
    llama = dict(SCOUT, num_hidden_layers=runs, hidden_size=d, num_attention_heads=nq, num_key_value_heads=nkv,
                 head_dim=kd, num_local_experts=E, num_experts_per_tok=top, intermediate_size=f,
                 intermediate_size_mlp=fd, moe_layers=list(range(1, runs)), vocab_size=V, tie_word_embeddings=True,
                 max_position_embeddings=8192)
    return mib, llama


def paposun_configs(size, runs=8):
    """A Paposun model of eight layers (a matrix memory without a feed-forward, an attention layer with a gelu feed-forward,
    an attention layer that reads the one before's keys and values, and so on: three memories, five attention layers of
    which two share) and a Llama 4 model of eight dense layers with the same width, heads, feed-forward width and
    vocabulary.  A memory has 8 heads with width / 16 key rows and width / 8 value columns; a chunk is longer than the
    measured contexts, so every earlier key is read."""
    name, d, nq, nkv, kd, vd, E, top, f, fs, fd, V = size
    rot = {"base": 500000.0, "dims": kd // 2, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}
    att = lambda src: dict({"heads": nq, "kv_heads": nkv, "dim": kd, "vdim": vd, "scale": kd ** -0.5, "mask": {"size": 8192}, "rot": rot},
                           **({} if src is None else {"kv_from": src}))
    mem = {"heads": 8, "dim": d // 16, "vdim": d // 8, "gate_cap": 10.0}
    ff = {"kind": "dense", "ff": fd}
    L = lambda t, m, mlp: {"type": t, "mixer": m, "mlp": mlp}
    pap = {"architecture": "Paposun", "vocab": V, "width": d, "max_positions": 8192, "norm": {"eps": 1e-5}, "residual_mult": 0.5,
           "logit_scale": 0.5,
           "layers": [L("mlstm", mem, None), L("attention", att(None), ff), L("attention", att(1), ff), L("mlstm", mem, None),
                      L("attention", att(None), ff), L("attention", att(4), ff), L("mlstm", mem, None), L("attention", att(None), ff)]}
    llama = dict(SCOUT, num_hidden_layers=runs, hidden_size=d, num_attention_heads=nq, num_key_value_heads=nkv,
                 head_dim=kd, num_local_experts=E, num_experts_per_tok=top, intermediate_size=f,
                 intermediate_size_mlp=fd, moe_layers=[], vocab_size=V, tie_word_embeddings=True,
                 max_position_embeddings=8192)
    return pap, llama


def gapevik_configs(size, runs=8):
    """A Gapevik model of eight layer runs (attention with a convolution on q, k, v and capped scores; latent attention
    through a window with sinks; the gated delta rule; the first attention layer's weights again; and so on: three
    attention runs on one set of weights, three latent layers, two delta layers, experts with two identity experts
    everywhere) and a Llama 4 model of eight layers with the same width, experts and vocabulary, whose attention has
    the heads of Gapevik's attention layers.  A latent row is kv_rank + rot_dim = 128 elements; chunk and window are
    longer than the measured contexts, so every earlier key is read.  A delta layer has width / 128 heads of 128 x 128
    on half as many q/k heads."""
    name, d, nq, nkv, kd, vd, E, top, f, fs, fd, V = size
    att = {"heads": nq, "kv_heads": nkv, "dim": kd, "vdim": kd, "scale": kd ** -0.5, "mask": {"size": 8192}, "softcap": 30.0,
           "conv": 4, "rot": {"base": 500000.0, "dims": kd // 2}}
    lat = {"heads": 16, "dim": 64, "rot_dim": 32, "vdim": 64, "q_rank": d // 4, "kv_rank": 96, "scale": 96 ** -0.5,
           "mask": {"size": 8192}, "rot": {"base": 20000.0, "dims": 32}}
    dlt = {"heads": d // 128, "kv_heads": d // 256, "dim": 128, "vdim": 128, "conv": 4}
    moe = {"kind": "moe", "expert": {"ff": f}, "router": {"experts": E, "identity": 2, "top": top}}
    L = lambda t, m, **kw: dict({"type": t, "mixer": m, "mlp": moe}, **kw)
    gap = {"architecture": "Gapevik", "vocab": V, "width": d, "max_positions": 8192, "norm": {"eps": 1e-6}, "residual_mult": 0.5,
           "embedding": {"scale": d ** 0.5},
           "layers": [L("attention", att), L("latent_attention", lat), L("delta", dlt), L("attention", att, weights_of=0),
                      L("latent_attention", lat), L("delta", dlt), L("attention", att, weights_of=0), L("latent_attention", lat)]}
    llama = dict(SCOUT, num_hidden_layers=runs, hidden_size=d, num_attention_heads=nq, num_key_value_heads=nkv,
                 head_dim=kd, num_local_experts=E, num_experts_per_tok=top, intermediate_size=f,
                 intermediate_size_mlp=fd, moe_layers=list(range(runs)), vocab_size=V, tie_word_embeddings=True,
                 max_position_embeddings=8192)
    return gap, llama


def zuzadra_configs(size, runs=8):
    """A Zuzadra model of eight layer runs (two state-space layers, the parallel layer of attention and decaying memory, one
    more state-space layer, all run twice on one set of weights) with four residual streams, and a Paposun model of eight
    layers (a matrix memory where Zuzadra has a state space, attention where it has the parallel layer) with the same
    width, attention heads, feed-forward width and vocabulary, a feed-forward in every layer of both.  A state space has
    width / 32 heads of 64 with 128 state rows, a decaying memory width / 64 heads of 64, a matrix memory 8 heads of width /
    16 key rows and width / 8 value columns; the window is longer than the measured contexts."""
    name, d, nq, nkv, kd, vd, E, top, f, fs, fd, V = size
    ff = {"kind": "dense", "ff": fd}
    L = lambda t, m: {"type": t, "mixer": m, "mlp": ff}
    ssm = {"heads": d // 32, "vdim": 64, "state": 128, "groups": 1, "conv": 4, "norm_groups": 1}
    par = {"left": {"heads": nq, "kv_heads": nkv, "dim": kd, "vdim": vd, "scale": kd ** -0.5, "mask": {"size": 8192},
                    "rot": {"base": 500000.0, "dims": kd // 2}},
           "right": {"heads": d // 64, "dim": 64, "rank": 64}, "left_scale": 0.75, "right_scale": 0.6}
    zuz = {"architecture": "Zuzadra", "vocab": V, "width": d, "max_positions": 8192, "norm": {"eps": 1e-6}, "streams": 4,
           "loop": {"start": 0, "stop": 4, "times": 2},
           "layers": [L("mamba2", ssm), L("mamba2", ssm), L("parallel", par), L("mamba2", ssm)]}
    mem = {"heads": 8, "dim": d // 16, "vdim": d // 8, "gate_cap": 10.0}
    att = {"heads": nq, "kv_heads": nkv, "dim": kd, "vdim": vd, "scale": kd ** -0.5, "mask": {"size": 8192},
           "rot": {"base": 500000.0, "dims": kd // 2}}
    pap = {"architecture": "Paposun", "vocab": V, "width": d, "max_positions": 8192, "norm": {"eps": 1e-6}, "residual_mult": 0.5,
           "logit_scale": 0.5,
           "layers": [L("mlstm", mem), L("mlstm", mem), L("attention", att), L("mlstm", mem)] * 2}
    return zuz, pap


def fozutar_configs(size, runs=8):
    """A Fozutar model of eight layer runs (gated linear attention, then attention and gated linear attention three times on
    one set of weights, then one more attention layer) and a Gapevik model of eight layers with a delta layer where Fozutar has
    gated linear attention and attention where it has attention, on the same sets of weights (the loop's layers borrow), with
    the same width, attention heads, chunk, cap, experts and vocabulary.  A gated linear attention has width / 128 heads of 64
    key and 128 value elements with a decay of inner size 16, a delta layer width / 128 heads of 128 x 128 on half as many
    q/k heads; the chunk is longer than the measured contexts, so every earlier key is read."""
    name, d, nq, nkv, kd, vd, E, top, f, fs, fd, V = size
    att = {"heads": nq, "kv_heads": nkv, "dim": kd, "vdim": kd, "scale": kd ** -0.5, "mask": {"size": 8192}, "softcap": 30.0}
    gla = {"heads": d // 128, "dim": 64, "vdim": 128, "tau": 16.0, "rank": 16}
    dlt = {"heads": d // 128, "kv_heads": d // 256, "dim": 128, "vdim": 128, "conv": 4}
    moe = lambda **more: {"kind": "moe", "expert": {"ff": f}, "router": dict(more, experts=E, top=top)}
    foz_att = dict(att, bias_max=4096, buckets=32)
    gap_att = dict(att, conv=4, rot={"base": 500000.0, "dims": kd // 2})
    L = lambda t, m, ff, **kw: dict({"type": t, "mixer": m, "mlp": ff}, **kw)
    common = {"vocab": V, "width": d, "max_positions": 8192, "norm": {"eps": 1e-6}, "embedding": {"scale": d ** 0.5}}
    foz = dict(common, architecture="Fozutar", loop={"start": 1, "stop": 3, "times": 3},
               layers=[L("gla", gla, moe()), L("attention", foz_att, moe()), L("gla", gla, moe()), L("attention", foz_att, moe())])
    A, D = (lambda **kw: L("attention", gap_att, moe(identity=0), **kw)), (lambda **kw: L("delta", dlt, moe(identity=0), **kw))
    gap = dict(common, architecture="Gapevik", residual_mult=0.5,
               layers=[D(), A(), D(), A(weights_of=1), D(weights_of=2), A(weights_of=1), D(weights_of=2), A()])
    return foz, gap


def design_work(model, T, contexts):
    """(flops of a prompt of T tokens, bytes a decode step over `contexts` must read), from the parts' own sizes
    as the design states them (no padding): every layer run reads its weights once; experts by the tokens' draw."""
    from spite_b200.config.specs import LayerCall
    from spite_b200.parts.feedforward import DenseActivation, MoESigmoidPrescaled, MoESoftmaxTopK
    from spite_b200.parts.latent import LatentAttention
    from spite_b200.parts.mlstm import MatrixLstm
    from spite_b200.parts.delta import GatedDelta
    from spite_b200.parts.gla import GatedLinearAttention
    from spite_b200.parts.parallel import ParallelMixers
    from spite_b200.parts.statespace import StateSpace
    es, p = 2, model.plan
    flops, nbytes = 2 * p.hidden_size * p.vocab_size, p.vocab_size * p.hidden_size * es
    for j in model.junctions:
        if j.kind == "reinject_add":                 # two sums a row: no product, no weights to speak of
            continue
        n = sum(1 for c in p.order if not isinstance(c, LayerCall))
        flops += n * 2 * T * 2 * j.d * j.d
        nbytes += n * 2 * j.d * j.d * es
    for call in p.layer_calls():
        blk = model.blocks[call.layer]
        m, d = blk.mixer, p.hidden_size
        if isinstance(m, LatentAttention):
            # the design's own count: keys and values of every head expanded from the latents (the products with the
            # heads' matrices are part of w), scores over head_dim + rotary_dim, values over value_dim; a decode step
            # reads one row of kv_rank + rotary_dim elements per cached position
            w = d * (m.rq + m.rkv + m.dr + m.nq) + m.rq * m.nq * (m.dn + m.dr) + m.nq * (m.dn + m.dv) * m.rkv + m.nq * m.dv * d
            flops += 2 * T * w + 2 * m.nq * (m.dn + m.dr + m.dv) * T * (T + 1) // 2
            nbytes += w * es + sum(c * (m.rkv + m.dr) * es for c in contexts)
        elif isinstance(m, MatrixLstm):
            # projections (q, k, v, the gate, the two gates of the recurrence) and the output; per token and head the
            # state's update and its read-out, two multiply-adds an element; a decode step reads and writes the state
            w = d * (2 * m.H * m.kd + 2 * m.H * m.vd + 2 * m.H) + m.H * m.vd * d
            flops += 2 * T * w + 4 * T * m.H * m.kd * m.vd
            nbytes += w * es + len(contexts) * 2 * m.H * (m.kd * m.vd + m.kd + 1) * 4
        elif isinstance(m, GatedDelta):
            # projections (q, k, v, the gate, two numbers a head) and the output; per token and head the matrix's decay
            # and correction and its read-out, two multiply-adds an element; a decode step reads and writes the matrices
            w = d * (2 * m.G * m.kd + 2 * m.H * m.vd + 2 * m.H) + m.H * m.vd * d
            flops += 2 * T * w + 4 * T * m.H * m.kd * m.vd
            nbytes += w * es + len(contexts) * 2 * m.H * m.kd * m.vd * 4
        elif isinstance(m, GatedLinearAttention):
            # projections (q, k, v, the gate, the decay's two) and the output; per token and head the matrix's update and its
            # read-out, two multiply-adds an element; a decode step reads and writes the matrices
            w = d * (2 * m.nk + 2 * m.nv + m.rank) + m.rank * m.nk + m.nv * d
            flops += 2 * T * w + 4 * T * m.H * m.kd * m.vd
            nbytes += w * es + len(contexts) * 2 * m.H * m.kd * m.vd * 4
        elif isinstance(m, StateSpace):
            # both projections; per token and head the matrix's update and its read-out, two multiply-adds an element
            w = d * (2 * m.inner + 2 * m.G * m.N + m.H) + m.inner * d
            flops += 2 * T * w + 4 * T * m.inner * m.N
            nbytes += w * es + len(contexts) * 2 * m.inner * m.N * 4
        elif isinstance(m, ParallelMixers):
            a, b = m.sides["left"], m.sides["right"]
            w = d * (a.nq * a.kd + a.nkv * (a.kd + a.vd)) + a.nq * a.vd * d + d * (4 * b.n + b.rank) + b.n * b.rank + b.n * d
            flops += 2 * T * w + 2 * a.nq * (a.kd + a.vd) * T * (T + 1) // 2 + 4 * T * b.n * b.dim
            nbytes += w * es + sum(c * a.nkv * (a.kd + a.vd) * es for c in contexts) + len(contexts) * 2 * b.n * b.dim * 4
        else:
            shared = getattr(m, "kv_shared", False)
            keys_alone = getattr(m, "values_are_keys", False)         # one row a position serves as key and value
            w = d * (m.nq * m.kd + (0 if shared else m.nkv * (m.kd + (0 if keys_alone else m.vd)))) + m.nq * m.vd * d + \
                (m.nq * d if getattr(m, "head_gate", False) else 0) + (m.nq * m.vd * d if getattr(m, "output_gate", False) else 0)
            flops += 2 * T * w + 2 * m.nq * (m.kd + m.vd) * T * (T + 1) // 2
            nbytes += w * es + sum(c * m.nkv * (m.kd + (0 if keys_alone else m.vd)) * es for c in contexts)
        f = blk.ffn
        if f is None:
            continue
        if isinstance(f, MoESoftmaxTopK):
            used = torch_unique(f)
            flops += 2 * T * d * (f.E + f.identity + 3 * f.top_k * f.f)
            nbytes += 3 * d * used * f.f * es + (f.E + f.identity) * d * 4
        elif isinstance(f, DenseActivation):
            flops += 2 * T * 2 * d * f.f
            nbytes += 2 * d * f.f * es
        elif isinstance(f, MoESigmoidPrescaled):
            mats = 3 if f.gated else 2
            used = torch_unique(f)
            flops += 2 * T * d * (f.E + mats * (f.top_k * f.f + f.fs))
            nbytes += (mats * d * (used * f.f + f.fs)) * es + f.E * d * 4
        else:
            flops += 2 * T * 3 * d * f.f
            nbytes += 3 * d * f.f * es
    return flops, nbytes


def torch_unique(ffn):
    import torch
    r = getattr(ffn, "last_routing", None)
    if r is None:
        return ffn.E
    ids = torch.unique(r.expert_ids)
    return int((ids < ffn.E).sum())                  # (identity experts have no weights to read)


def run_sezazen(args):
    """A design (`--config sezazen`, `mibezen` or `paposun`) beside the closest existing one, Llama 4, at equal layer sizes:
    prefill of 2,048 tokens (a fraction of the sustained bf16 rate) and decode at batch 1 and 8 with 2,048 cached
    tokens (a fraction of the copy bandwidth).  One JSON line; `value` is the design's decode rate at batch 8 at
    the first size."""
    design = args.config
    configs_of = {"sezazen": design_configs, "mibezen": mibezen_configs, "paposun": paposun_configs,
                  "gapevik": gapevik_configs, "zuzadra": zuzadra_configs, "fozutar": fozutar_configs}[design]
    other = {"zuzadra": "paposun", "fozutar": "gapevik"}.get(design, "llama4")
    import torch
    from spite_b200.config import config_from_dict
    from spite_b200.engine import Engine, Model, StepEntry
    from spite_b200.kernels import build as kb
    torch.cuda.set_device(0)
    pk, pk_src = peaks()
    T, C, steps, warmup = 2048, 2048, args.steps if args.only_decode else max(args.steps, 16), max(args.warmup, 3)
    out, launches, clocks = {}, 0, ClockSampler()

    def measure(cfgd):
        nonlocal launches
        cfg = config_from_dict(cfgd)
        model = Model.from_config(cfg, dtype="bfloat16", device="cuda:0")
        kb.ensure_built(model.kernel_libraries() + ["sampling"])
        model.init_random(seed=0, std=0.02)
        ks, V = model.kernels, model.plan.vocab_size
        engine = Engine(model, cache_tokens=9 * (C + 256), page_size=64, max_requests=9,
                        cuda_graphs=False if args.no_graphs else None)
        g = torch.Generator().manual_seed(5)
        res = {}
        # prefill: one prompt of T tokens, its last position's logits; a new request every time
        ms = []
        for i in range(0 if args.only_decode else warmup + 5):
            toks = torch.randint(0, V, (T,), generator=g).tolist()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            engine.step([StepEntry("p", toks, [T - 1])])
            e1.record()
            torch.cuda.synchronize()
            engine.finish("p")
            if i >= warmup:
                ms.append(e0.elapsed_time(e1))
        if ms:
            pre = sorted(ms)[len(ms) // 2]
            flops, _ = design_work(model, T, [])
            res.update(prefill_ms=round(pre, 3), prefill_tok_s=round(T * 1e3 / pre), prefill_tflops=round(flops / pre / 1e9, 1),
                       prefill_frac=round(flops / (pre * 1e-3) / (pk["bf16_tflops_sustained"] * 1e12), 3))
        for B in ((args.batch,) if args.only_decode else (1, 8)):
            if args.only_prefill:
                break
            rids = [f"d{B}_{i}" for i in range(B)]
            for r in rids:
                engine.step([StepEntry(r, torch.randint(0, V, (C,), generator=g).tolist(), [])])
            ids = torch.randint(0, V, (steps + warmup, B), generator=g).tolist()
            for i in range(warmup):
                ks.argmax(engine.step([StepEntry(r, [ids[i][j]], [0]) for j, r in enumerate(rids)]))
            torch.cuda.synchronize()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            for i in range(warmup, warmup + steps):
                ks.argmax(engine.step([StepEntry(r, [ids[i][j]], [0]) for j, r in enumerate(rids)]))
            e1.record()
            torch.cuda.synchronize()
            dms = e0.elapsed_time(e1) / steps
            _, nbytes = design_work(model, 1, [engine.cached_tokens(r) for r in rids])
            res.update({f"decode_b{B}_ms": round(dms, 4), f"decode_b{B}_tok_s": round(B * 1e3 / dms, 1),
                        f"decode_b{B}_gb": round(nbytes / 1e9, 3),
                        f"decode_b{B}_hbm_frac": round(nbytes / (dms * 1e-3) / (pk["hbm_gbs"] * 1e9), 3)})
            for r in rids:
                engine.finish(r)
        engine.check()
        launches += ks.launches
        res["weights_gb"] = round(model.weight_bytes() / 1e9, 2)
        del engine, model
        torch.cuda.empty_cache()
        return res

    sizes = [s for s in (DESIGN_SIZES if design == "sezazen" else DESIGN_SIZES[:2]) if args.size in (None, s[0])]
    with clocks:
        for size in sizes:
            sez, llama = configs_of(size)
            out[size[0]] = {name: measure(cfgd) for name, cfgd in ((design, sez), (other, llama))
                            if args.design in ("both", name)}
    first = next(iter(out[sizes[0][0]].values()))
    key = f"decode_b{args.batch if args.only_decode else 8}"
    line = base_line(f"decode tok/s at batch 8, context 2,048 ({design.capitalize()} design, first size)", first.get(key + "_tok_s", 0.0), "tok/s",
                     steps, warmup, first.get(key + "_ms", 0.0),
                     {"model": f"{design} beside {other} at equal layer sizes", "layer_runs": 8, "prefill_tokens": T, "context": C,
                      "sizes": {s[0]: dict(zip(("width", "q_heads", "kv_heads", "key_dim", "value_dim", "experts", "top", "expert_ff",
                                                "shared_ff", "dense_ff", "vocab"), s[1:])) for s in DESIGN_SIZES},
                      "global_batch": 8, "seq_len": C, "page_size": 64, "parallelism": "single-gpu",
                      "l2": "inputs larger than L2 (the weights a step reads exceed 126 MB)"})
    line.update({"gpu_launches": launches, "clocks": clocks.summary(), "peaks": dict(pk, source=pk_src), "designs": out})
    print(json.dumps(line))


def run_ours(args):
    import torch
    from spite_b200.engine import Engine, StepEntry
    from spite_b200.engine.scheduler import Request, Scheduler
    from spite_b200.sampling import Sampler, SamplingParams

    dev = "cuda:0"
    cfgd = dict(SCOUT, num_hidden_layers=args.layers)
    cfg, model = build_model(cfgd)
    ks = model.kernels
    B, ctx = args.batch, args.context
    page = 64
    max_b = max(B, 64 if not args.skip_points else B)
    engine = Engine(model, cache_tokens=max_b * (ctx + page), page_size=page, max_requests=max_b,
                    max_positions=ctx + page, cuda_graphs=False if args.no_graphs else None)
    for kv in engine.storage.kv:                       # a cache as earlier steps would have left it
        kv.normal_(0.0, 1.0)
    g = torch.Generator().manual_seed(1)
    vocab = cfg.vocab_size

    def occupy(n_req, n_cached):
        for r in list(engine.cache.requests):
            engine.finish(r)
        for r in range(n_req):
            engine.cache.admit(r)
            engine.cache.reserve(r, n_cached)
            engine.cache.commit(r)

    def timed_decode(n_req, steps, warmup, clocks=None):
        start_ctx = ctx - (steps + warmup) - 1
        occupy(n_req, start_ctx)
        toks = torch.randint(0, vocab, (steps + warmup, n_req), generator=g).tolist()
        ids = None
        for i in range(warmup):
            ids = ks.argmax(engine.step([StepEntry(r, [toks[i][r]], [0]) for r in range(n_req)]))
        torch.cuda.synchronize()
        l0 = ks.launches
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        ctxm = clocks if clocks is not None else _Null()
        with ctxm:
            e0.record()
            for i in range(warmup, warmup + steps):
                ids = ks.argmax(engine.step([StepEntry(r, [toks[i][r]], [0]) for r in range(n_req)]))
            e1.record()
            torch.cuda.synchronize()
        ms = e0.elapsed_time(e1)
        return ms / steps, ks.launches - l0, ids

    pk, pk_src = peaks()
    def measure_prefill():
        """Prefill of 2,048 tokens, logits of the last row."""
        T = 2048
        ptoks = torch.randint(0, vocab, (T,), generator=g).tolist()
        pre_ms = []
        for i in range(6):
            torch.cuda.synchronize()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            engine.step([StepEntry("p", ptoks, [T - 1])])
            e1.record()
            torch.cuda.synchronize()
            engine.finish("p")
            pre_ms.append(e0.elapsed_time(e1))
        pms = sorted(pre_ms[1:])[2]                       # the median of five runs after one warm-up
        pflops = prefill_flops(cfgd, T)
        if args.verbose:
            print("prefill runs (ms):", [round(x, 2) for x in pre_ms], file=sys.stderr)
        floor = prefill_roofline_ms(cfgd, T, pk)
        # frac: the step's flops / time / the sustained bf16 peak.  frac_kernel_roofline: the time the step's kernels
        # cannot beat one by one (the experts' weights make their products memory-bound at this length) / time
        return {"value": round(T * 1000.0 / pms, 1), "tokens": T, "ms": round(pms, 3),
                "frac": round(pflops / (pms * 1e-3) / (pk["bf16_tflops_sustained"] * 1e12), 4),
                "roofline_ms": round(floor, 3), "frac_kernel_roofline": round(floor / pms, 4)}

    if args.only_prefill:
        print(json.dumps({"prefill": measure_prefill(), "layers": args.layers}))
        return
    clocks = ClockSampler()
    ms_step, launches, _ = timed_decode(B, args.steps, args.warmup, clocks)
    value = B * 1000.0 / ms_step
    def step_bytes(n_req):
        """Bytes a decode step of `n_req` requests at the end of the context has to read; the experts its tokens
        use, layer by layer, are the mean over a few more (untimed) steps of the same kind."""
        probe = 8
        occupy(n_req, ctx - probe - 1)
        ptoks = torch.randint(0, vocab, (probe, n_req), generator=g).tolist()
        distinct = [0.0] * len(model.blocks)
        for i in range(probe):
            engine.step([StepEntry(r, [ptoks[i][r]], [0]) for r in range(n_req)])
            for li, n in enumerate(distinct_experts(model)):
                distinct[li] += n / probe
        return decode_bytes(model, engine, [ctx - 1] * n_req, distinct)
    nbytes = step_bytes(B)
    achieved = nbytes / (ms_step * 1e-3) / 1e9
    engine.check()
    if args.only_decode:
        print(json.dumps({"decode_ms_per_step": round(ms_step, 4), "tok_per_s": round(value, 1), "batch": B,
                          "layers": args.layers, "launches": launches, "GBps": round(achieved, 1)}))
        return

    # end to end through the scheduler: host tokens in (pinned copy), sampled tokens out
    sched = Scheduler(engine, Sampler(ks), max_batch_tokens=4096, ctx=ctx + page)
    occupy(B, ctx - (args.steps + args.warmup) - 2)
    prompt_tail = torch.randint(0, vocab, (B,), generator=g).tolist()
    for r in range(B):
        req = Request(r, [0] * engine.cached_tokens(r) + [prompt_tail[r]],
                      SamplingParams(temperature=0.0, max_tokens=args.steps + args.warmup + 1))
        req.n_fed = engine.cached_tokens(r)
        req.state = req.state.__class__.PREFILLING
        req.rng_state = 0
        sched.running.append(req)
    for _ in range(args.warmup + 1):
        sched.step()
    torch.cuda.synchronize()
    t0 = time.perf_counter()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    n_tok = 0
    for _ in range(args.steps - 1):
        n_tok += sum(1 for o in sched.step() if o.token is not None)
    e1.record()
    torch.cuda.synchronize()
    e2e_ms = max(e0.elapsed_time(e1), (time.perf_counter() - t0) * 1e3)
    e2e = n_tok * 1000.0 / e2e_ms if e2e_ms > 0 else 0.0
    table_w = -(-(ctx + page) // page)
    h2d = 4 * (3 * B + (B + 1) + B + B + 2 * B * table_w)
    for r in list(engine.cache.requests):
        engine.finish(r)

    points = {}
    if not args.skip_points:
        for nb in (1, 64):
            pc = ClockSampler()
            # long enough for the clock sampler to see it: a step of one token takes a few milliseconds
            ms_b, _, _ = timed_decode(nb, max(4, args.steps * 4 if nb == 1 else args.steps // 2), 3, pc)
            gbs = step_bytes(nb) / (ms_b * 1e-3) / 1e9
            # each point with its own step time, fraction of the HBM roofline and clocks (flat: the record keeps one level)
            points.update({f"decode_b{nb}": round(nb * 1000.0 / ms_b, 1), f"decode_b{nb}_ms": round(ms_b, 4),
                           f"decode_b{nb}_GBps": round(gbs, 1), f"decode_b{nb}_hbm_frac": round(gbs / pk["hbm_gbs"], 4),
                           f"decode_b{nb}_sm_mhz": pc.summary()["sm_mhz"]})
        for r in list(engine.cache.requests):
            engine.finish(r)
    engine.check()

    prefill = measure_prefill()
    engine.check()

    line = {
        "metric": f"decode tok/s (Llama-4-Scout-shaped, batch {B}, context {ctx})",
        "value": round(value, 2), "unit": "tok/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
        "ms_per_step": round(ms_step, 4), "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic (random token ids, random weights N(0,0.02))",
        "config": {"model": "llama4-scout-shaped", "layers": args.layers, "layers_full": FULL_LAYERS,
                   "hidden": 5120, "q_heads": 40, "kv_heads": 8, "head_dim": 128, "experts": 16, "top_k": 1,
                   "expert_ffn": 8192, "shared_ffn": 8192, "vocab": 202048, "chunk": 8192, "nope_every": 4,
                   "global_batch": B, "seq_len": ctx, "page_size": page, "parallelism": "single-gpu",
                   "l2": "inputs larger than L2 (weights read per step exceed 126 MB)",
                   "cache": "random-filled to context"},
        "e2e": {"value": round(e2e, 2), "unit": "tok/s", "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": 4 * B,
                "ids_read": "one step late (decode steps are launched from the ids on the device)"
                if sched.counters["steps_ahead"] else "every step"},
        "gpu_launches": launches,
        "clocks": clocks.summary(),
        "prefill": prefill,
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4), "bytes_per_step": nbytes, "peaks": pk_src},
        "points": points,
    }
    print(json.dumps(line))


class _Null:
    def __enter__(self):
        return self

    def __exit__(self, *a):
        return False


def run_reference(args):
    # giveen/spite is a Rust workspace (Cargo.toml, no pyproject/setup.py): pip cannot install it, the
    # image has no cargo/rustc, and its Llama 4 path has no GPU kernel to run.
    print(json.dumps({"impl": "reference",
                      "unavailable": "giveen/spite is a Rust workspace without a Python package; "
                                     "no cargo/rustc offline, and its Llama 4 path is CPU-only"}))
    return 0


def main(argv=None):
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--impl", choices=["ours", "reference"], default="ours")
    ap.add_argument("--config", choices=["scout", "maverick", "long", "sezazen", "mibezen", "paposun", "gapevik", "zuzadra", "fozutar"], default="scout",
                    help="scout: the benchmark line; maverick, long, sezazen, mibezen, paposun, gapevik, zuzadra, fozutar: further workloads, one line each")
    ap.add_argument("--layers", type=int, default=FULL_LAYERS)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--context", type=int, default=8192)
    ap.add_argument("--skip-points", action="store_true")
    ap.add_argument("--no-graphs", action="store_true", help="launch every kernel of a decode step by itself")
    ap.add_argument("--only-decode", action="store_true", help="measure the decode step only (for profiling)")
    ap.add_argument("--only-prefill", action="store_true", help="measure the prefill step only (for profiling)")
    ap.add_argument("--verbose", action="store_true", help="print the single prefill timings to standard error")
    ap.add_argument("--size", default=None, help="--config sezazen: only this set of layer sizes (small, medium, ...)")
    ap.add_argument("--design", choices=["both", "sezazen", "mibezen", "paposun", "gapevik", "zuzadra", "fozutar", "llama4"], default="both",
                    help="--config sezazen / mibezen / paposun / gapevik / zuzadra / fozutar: only this design")
    args = ap.parse_args(argv)
    if args.impl == "reference":
        return run_reference(args)
    if args.gpus != 1:
        print(f"bench.py measures one GPU; --gpus {args.gpus} is not supported by this engine")
        return 2
    if args.config == "maverick":
        run_maverick(args)
        return 0
    if args.config == "long":
        run_long(args)
        return 0
    if args.config in ("sezazen", "mibezen", "paposun", "gapevik", "zuzadra", "fozutar"):
        run_sezazen(args)
        return 0
    if args.warmup < 3:
        args.warmup = 3
    if args.steps < 1 or args.steps + args.warmup + 16 > args.context:
        print(f"bench.py: --steps {args.steps} with --warmup {args.warmup} does not fit the context of {args.context}")
        return 2
    run_ours(args)
    return 0


if __name__ == "__main__":
    sys.exit(main())
