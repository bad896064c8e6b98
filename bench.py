#!/usr/bin/env python3
"""Benchmark of the engine on one B200: decode tokens per second at the Qwen3-8B shape
(random bfloat16 weights, batch 8, 2048-token prompts, 16-token cache pages), with the
prefill rate of one 2048-token prompt, decode at batch 1 and 64, the same decode
measured end to end through the Python entry point, and roofline fractions.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl ours|reference]

A "step" is one decode step of the whole batch.  Prints one JSON line.
"""
from __future__ import annotations

import argparse
import json
import os
import random
import statistics
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

# the headline configuration: the Qwen3-8B shape
SHAPE = dict(num_layers=36, hidden_size=4096, num_heads=32, num_kv_heads=8, head_dim=128,
             intermediate_size=12288, vocab_size=151936, rope_theta=1e6, rms_norm_eps=1e-6, max_position=40960)
CONTEXT = 4096
PROMPT_LEN = 2048
PAGE_SIZE = 16
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0}


def load_peaks():
    p = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.isfile(p):
        try:
            with open(p) as f:
                d = json.load(f)
            out = dict(FALLBACK_PEAKS)
            for k in out:
                if isinstance(d.get(k), (int, float)) and d[k] > 0:
                    out[k] = float(d[k])
            out["source"] = "measured"
            return out
        except Exception:
            pass
    out = dict(FALLBACK_PEAKS)
    out["source"] = "fallback"
    return out


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while a region runs."""
    Q = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
         "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.samples = []
        self.proc = None
        self.thread = None

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", "0", f"--query-gpu={self.Q}", "--format=csv,noheader,nounits",
                                          "-lms", "50"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
        except OSError:
            self.proc = None
            return

        def pump():
            for line in self.proc.stdout:
                self.samples.append(line.strip())
        self.thread = threading.Thread(target=pump, daemon=True)
        self.thread.start()

    def stop(self):
        if self.proc is not None:
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except Exception:
                self.proc.kill()

    def summary(self):
        sm, mx, reasons = [], [], set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for s in self.samples:
            f = [x.strip() for x in s.split(",")]
            if len(f) < 6:
                continue
            try:
                sm.append(float(f[0])); mx.append(float(f[1]))
            except ValueError:
                continue
            for n, v in zip(names, f[2:6]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        if not sm:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": [], "samples": 0}
        return {"sm_mhz": statistics.median(sm), "sm_max_mhz": max(mx), "reasons": sorted(reasons), "samples": len(sm)}


def make_engine(layers: int, max_live: int, cache_tokens: int, seed: int = 0, graphs: bool = True,
                context: int = CONTEXT, step_tokens: int = PROMPT_LEN):
    import torch
    import tffinfer_b200 as tff
    from tffinfer_b200.config import Qwen3Config
    from tffinfer_b200.weights import random_tensors_on_device
    cfg = Qwen3Config(architecture="Qwen3ForCausalLM", tie_word_embeddings=False,
                      layer_types=("full_attention",) * layers, **{**SHAPE, "num_layers": layers}).validate()
    tensors = random_tensors_on_device(cfg, seed, "cuda", "bfloat16")
    ecfg = tff.EngineConfig(dtype="bfloat16", page_size=PAGE_SIZE, max_cache_tokens=cache_tokens,
                            max_live_requests=max_live, max_tokens_per_step=step_tokens, max_model_len=context,
                            use_cuda_graphs=graphs)
    runner = tff.ModelRunner(config=cfg, tensors=tensors, engine_config=ecfg)
    del tensors
    torch.cuda.empty_cache()
    return tff.Engine(runner=runner), cfg


def model_bytes(cfg) -> dict:
    H, L, I, V = cfg.hidden_size, cfg.num_layers, cfg.intermediate_size, cfg.vocab_size
    qw, kvw = cfg.num_heads * cfg.head_dim, cfg.num_kv_heads * cfg.head_dim
    per_layer = (qw + 2 * kvw) * H + H * qw + 3 * I * H
    return {"layer_params": per_layer, "weights_read_per_step": 2 * (per_layer * L + V * H),
            "kv_bytes_per_token": 2 * L * cfg.num_kv_heads * cfg.head_dim * 2}


def decode_run(engine, batch: int, steps: int, warmup: int, seed: int, sampler=None, prompt_len: int = PROMPT_LEN):
    """Prefills ``batch`` prompts of ``prompt_len`` tokens, then times ``steps`` decode steps
    after ``warmup`` untimed ones.  Returns device-timed and wall-clock figures."""
    import torch
    from tffinfer_b200 import SamplingParams
    rng = random.Random(seed)
    vocab = engine.runner.desc.vocab_size
    # earlier requests decode while later ones prefill, a step's token budget at a time
    budget = max(1, engine.runner.ecfg.max_tokens_per_step)
    sp = SamplingParams(max_new_tokens=warmup + steps + 8 + batch * -(-prompt_len // budget))
    ids = [engine.add_request([rng.randrange(vocab) for _ in range(prompt_len)], sp,
                              request_id=f"b{batch}_{prompt_len}_{i}", key=i)
           for i in range(batch)]
    # prefill: until every request has produced its first token
    while any(len(engine.requests[i].generated) == 0 for i in ids):
        engine.step()
    for _ in range(warmup):
        engine.step()
    torch.cuda.synchronize()
    ops = engine.runner.ops
    launches0 = ops.launches
    ctx0 = sum(len(engine.requests[i]) for i in ids) / batch
    ev = [(torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)) for _ in range(steps)]
    engine.step_events = None
    if sampler is not None:
        sampler.start()
    t0 = time.perf_counter()
    for k in range(steps):
        engine.step_events = ev[k]
        outs = engine.step()
        assert len(outs) == batch
    torch.cuda.synchronize()
    wall = time.perf_counter() - t0
    if sampler is not None:
        sampler.stop()
    engine.step_events = None
    per_step = sorted(a.elapsed_time(b) for a, b in ev)
    dev_ms = sum(per_step)
    ctx1 = sum(len(engine.requests[i]) for i in ids) / batch
    launches = ops.launches - launches0
    ops.check_errors()
    h2d = engine.runner.last_h2d_bytes
    # (the newest tokens have not been read back yet)
    last_tokens = [engine.requests[i].generated[-min(4, len(engine.requests[i].generated))] for i in ids]
    for i in ids:                                   # stop the requests and give their pages back
        engine.abort(i)
    return {"tok_s": batch * steps / (dev_ms / 1e3), "ms_per_step": dev_ms / steps,
            "e2e_tok_s": batch * steps / wall, "launches": launches, "last_tokens": last_tokens, "mean_context": (ctx0 + ctx1) / 2,
            "h2d_bytes": h2d, "d2h_bytes": 4 * batch + 4,      # drawn tokens and the kernels' error word
            "p50_ms": per_step[len(per_step) // 2], "p99_ms": per_step[min(len(per_step) - 1, int(0.99 * len(per_step)))],
            "max_ms": per_step[-1]}


def prefill_run(engine, iters: int, warmup: int, seed: int, prompt_len: int = PROMPT_LEN):
    import torch
    from tffinfer_b200 import StepEntry
    rng = random.Random(seed)
    vocab = engine.runner.desc.vocab_size
    runner = engine.runner
    times = []
    for it in range(warmup + iters):
        toks = [rng.randrange(vocab) for _ in range(prompt_len)]
        rid = f"prefill{prompt_len}_{it}"
        runner.add_request(rid)
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        batch = runner.make_batch([StepEntry(rid, toks, [prompt_len - 1])])
        torch.cuda.synchronize()
        a.record()
        logits = runner.run_batch(batch)
        b.record()
        torch.cuda.synchronize()
        runner.cache.commit(rid, prompt_len)
        runner.finish_request(rid)
        if it >= warmup:
            times.append(a.elapsed_time(b))
        assert logits.shape[0] == 1
    runner.ops.check_errors()
    return statistics.median(times)


# whole-workload runs through the scheduler (a 14B shape with mixed prompts, a 32B shape with long prompts)
WORKLOADS = {
    "mixed14b": dict(shape=dict(num_layers=40, hidden_size=5120, num_heads=40, num_kv_heads=8, head_dim=128,
                                intermediate_size=17408, vocab_size=151936, rope_theta=1e6, rms_norm_eps=1e-6,
                                max_position=40960),
                     requests=32, prompt_lens=(128, 4096), new_tokens=128, chunk=512, context=4352),
    "long32b": dict(shape=dict(num_layers=64, hidden_size=5120, num_heads=64, num_kv_heads=8, head_dim=128,
                               intermediate_size=25600, vocab_size=151936, rope_theta=1e6, rms_norm_eps=1e-6,
                               max_position=40960),
                    requests=16, prompt_lens=(8192, 8192), new_tokens=256, chunk=2048, context=8448),
    # many short requests: 512 prompts of 64 to 512 tokens, 64 new tokens each, at most 256 live at a time
    "chat8b": dict(shape=dict(SHAPE), requests=512, prompt_lens=(64, 512), new_tokens=64, chunk=2048, context=1024, live=256),
    # the headline shape in true 32-bit (FFMA products, float32 attention and cache) on short prompts
    "fp32_short": dict(shape=dict(SHAPE), requests=4, prompt_lens=(64, 192), new_tokens=16, chunk=256, context=512,
                       dtype="float32"),
}


def run_workload(name: str, layers: int = 0) -> int:
    """Runs a whole workload (prompts prefilled in portions while others decode) and prints its totals."""
    import torch
    import tffinfer_b200 as tff
    from tffinfer_b200.config import Qwen3Config
    from tffinfer_b200.weights import random_tensors_on_device
    w = WORKLOADS[name]
    shape = dict(w["shape"])
    if layers:
        shape["num_layers"] = layers
    cfg = Qwen3Config(architecture="Qwen3ForCausalLM", tie_word_embeddings=False,
                      layer_types=("full_attention",) * shape["num_layers"], **shape).validate()
    rng = random.Random(0)
    lens = [rng.randint(*w["prompt_lens"]) for _ in range(w["requests"])]
    live = w.get("live", w["requests"])
    cache_tokens = sum(sorted((-(-(n + w["new_tokens"] + 1) // PAGE_SIZE) * PAGE_SIZE for n in lens), reverse=True)[:live])
    dtype = w.get("dtype", "bfloat16")
    ecfg = tff.EngineConfig(dtype=dtype, page_size=PAGE_SIZE, max_cache_tokens=cache_tokens,
                            max_live_requests=live, max_tokens_per_step=w["chunk"], max_model_len=w["context"])
    tensors = random_tensors_on_device(cfg, 0, "cuda", dtype)
    engine = tff.Engine(runner=tff.ModelRunner(config=cfg, tensors=tensors, engine_config=ecfg))
    del tensors
    torch.cuda.empty_cache()
    sp = tff.SamplingParams(max_new_tokens=w["new_tokens"])
    warm = engine.generate([[1, 2, 3, 4]], tff.SamplingParams(max_new_tokens=4))       # builds kernels, first graphs
    prompts = [[rng.randrange(cfg.vocab_size) for _ in range(n)] for n in lens]
    torch.cuda.synchronize()
    t0 = time.perf_counter()
    ids = [engine.add_request(p, sp, key=i) for i, p in enumerate(prompts)]
    steps = 0
    first_token_at = {}
    step_s = []
    while engine.has_unfinished():
        t_step = time.perf_counter()
        for o in engine.step():
            if o.token is not None and o.request_id not in first_token_at:
                first_token_at[o.request_id] = time.perf_counter() - t0
        step_s.append(time.perf_counter() - t_step)       # host time of a step: with steps launched ahead, the
        steps += 1                                        # device time of the step before
    step_s.sort()
    torch.cuda.synchronize()
    dt = time.perf_counter() - t0
    engine.runner.ops.check_errors()
    gen = sum(len(engine.requests[i].generated) for i in ids)
    st = engine.stats()
    print(json.dumps({"workload": name, "layers": cfg.num_layers, "requests": len(ids), "prompt_tokens": sum(lens),
                      "generated_tokens": gen, "seconds": round(dt, 3), "steps": steps,
                      "total_tok_s": round((sum(lens) + gen) / dt, 1), "generated_tok_s": round(gen / dt, 1),
                      "step_ms_p50": round(1e3 * step_s[len(step_s) // 2], 3),
                      "step_ms_p99": round(1e3 * step_s[min(len(step_s) - 1, int(0.99 * len(step_s)))], 3),
                      "mean_time_to_first_token_s": round(sum(first_token_at.values()) / max(1, len(first_token_at)), 3),
                      "pages_high_water": st["pages_high_water"], "pages_total": st["pages_total"],
                      "preemptions": st["preemptions"], "dtype": "bf16" if dtype == "bfloat16" else "fp32",
                      "data": "synthetic"}))
    return 0


# decode and prefill of the headline shape at other batch sizes and context lengths than the headline's
SWEEP_DECODE = [(1, 512), (1, 8192), (1, 32768), (8, 512), (8, 8192), (8, 32768), (64, 512), (64, 8192), (256, 1024)]
SWEEP_PREFILL = [512, 1024, 4096, 8192]


def prefill_flops(cfg, mb, T: int) -> float:
    """Products of the layers for T tokens, the causal half of the attention's two products, the output matrix
    for the one wanted row."""
    return (2 * T * mb["layer_params"] * cfg.num_layers
            + 2 * T * T * cfg.head_dim * cfg.num_heads * cfg.num_layers + 2 * cfg.vocab_size * cfg.hidden_size)


def run_sweep(layers: int, steps: int, warmup: int) -> int:
    """One JSON line a point: decode steps (bytes that must be read / time / measured copy rate) and whole-prompt
    prefill steps (flops / time / measured product rate) of the Qwen3-8B shape at further sizes."""
    import torch
    peaks = load_peaks()
    steps = min(steps, 24)
    need = max(b * (n + warmup + steps + 72 + b * -(-n // max(SWEEP_PREFILL))) for b, n in SWEEP_DECODE)
    engine, cfg = make_engine(layers, max(b for b, _ in SWEEP_DECODE), need, context=SHAPE["max_position"],
                              step_tokens=max(SWEEP_PREFILL + [PROMPT_LEN]))
    mb = model_bytes(cfg)
    for b, n in SWEEP_DECODE:
        run = decode_run(engine, b, steps, warmup, seed=10 + b, prompt_len=n)
        byts = mb["weights_read_per_step"] + b * run["mean_context"] * mb["kv_bytes_per_token"]
        print(json.dumps({"point": "decode", "batch": b, "context": round(run["mean_context"]), "layers": cfg.num_layers,
                          "tok_s": round(run["tok_s"], 1), "ms_per_step": round(run["ms_per_step"], 4),
                          "p99_ms": round(run["p99_ms"], 4), "gbytes_per_step": round(byts / 1e9, 2),
                          "hbm_frac": round(byts / (run["ms_per_step"] / 1e3) / 1e9 / peaks["hbm_gbs"], 4),
                          "peaks": peaks["source"]}), flush=True)
    for T in SWEEP_PREFILL:
        pms = prefill_run(engine, iters=3, warmup=2, seed=T, prompt_len=T)
        fl = prefill_flops(cfg, mb, T)
        print(json.dumps({"point": "prefill", "tokens": T, "layers": cfg.num_layers, "ms": round(pms, 3),
                          "tok_s": round(T / (pms / 1e3), 1), "tflops": round(fl / (pms / 1e3) / 1e12, 1),
                          "frac": round(fl / (pms / 1e3) / (peaks["bf16_tflops"] * 1e12), 4),
                          "frac_sustained": round(fl / (pms / 1e3) / (peaks["bf16_tflops_sustained"] * 1e12), 4),
                          "peaks": peaks["source"]}), flush=True)
    torch.cuda.synchronize()
    return 0


# layer sizes of other models of the family (layers, hidden, query heads, feed-forward; 8 key/value heads of 128 all)
OTHER_SHAPES = {"0.6B": (28, 1024, 16, 3072), "1.7B": (28, 2048, 16, 6144), "4B": (36, 2560, 32, 9728),
                "14B": (40, 5120, 40, 17408), "32B": (64, 5120, 64, 25600)}


def run_shapes(steps: int, warmup: int) -> int:
    """Decode at batch 1 and 8 (2048-token prompts) and a 2048-token prefill at the layer sizes of the other
    models of the family, one JSON line a shape: small models are bound by the latency of a layer's chain of
    kernels, large ones by their bytes."""
    import torch
    peaks = load_peaks()
    steps = min(steps, 24)
    for name, (layers, hidden, heads, inter) in OTHER_SHAPES.items():
        SHAPE.update(num_layers=layers, hidden_size=hidden, num_heads=heads, intermediate_size=inter)
        engine, cfg = make_engine(layers, 8, 8 * (PROMPT_LEN + warmup + steps + 96))
        mb = model_bytes(cfg)
        line = {"point": "shape", "model": f"Qwen3-{name} shape", "layers": layers, "hidden": hidden, "heads": heads,
                "intermediate": inter, "peaks": peaks["source"]}
        for b in (1, 8):
            run = decode_run(engine, b, steps, warmup, seed=b)
            byts = mb["weights_read_per_step"] + b * run["mean_context"] * mb["kv_bytes_per_token"]
            line[f"decode_b{b}"] = {"tok_s": round(run["tok_s"], 1), "ms_per_step": round(run["ms_per_step"], 4),
                                    "hbm_frac": round(byts / (run["ms_per_step"] / 1e3) / 1e9 / peaks["hbm_gbs"], 4)}
        pms = prefill_run(engine, iters=3, warmup=2, seed=4)
        fl = prefill_flops(cfg, mb, PROMPT_LEN)
        line["prefill"] = {"tokens": PROMPT_LEN, "ms": round(pms, 3), "tok_s": round(PROMPT_LEN / (pms / 1e3), 1),
                           "frac": round(fl / (pms / 1e3) / (peaks["bf16_tflops"] * 1e12), 4)}
        print(json.dumps(line), flush=True)
        del engine
        torch.cuda.empty_cache()
    return 0


ATTN_DECODE_POINTS = [(1, 529), (1, 8209), (1, 32785), (8, 529), (8, 2069), (8, 8213), (64, 531), (64, 2069), (256, 1057)]


def run_attn_decode(iters: int = 50) -> int:
    """The decode attention of the headline shape alone (one layer's cache, scattered pages, one new token a request):
    one JSON line a point with the time of a call (its kernel and the merge of the key shares), L2 flushed between
    calls, against the bytes of keys and values at the measured copy rate."""
    import math
    import numpy as np
    import torch
    from tffinfer_b200.engine.batch import StepBatch
    from tffinfer_b200.kernels.library import CudaKernels
    ops = CudaKernels()
    peaks = load_peaks()
    nq, nkv, d, page = SHAPE["num_heads"], SHAPE["num_kv_heads"], SHAPE["head_dim"], PAGE_SIZE
    dev = "cuda"
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
    for B, ctx in ATTN_DECODE_POINTS:
        rng = random.Random(B * 100003 + ctx)
        blocks = -(-(ctx + 1) // page)
        ids = list(range(B * blocks + 5))
        rng.shuffle(ids)
        table = torch.tensor([ids[i * blocks:(i + 1) * blocks] for i in range(B)], dtype=torch.int32, device=dev)
        cache = torch.randn((len(ids), 1, 2, nkv, page, d), device=dev, dtype=torch.bfloat16)
        q = torch.randn((B, nq * d), device=dev, dtype=torch.bfloat16)
        out = torch.empty_like(q)
        ar = torch.arange(B + 1, dtype=torch.int32, device=dev)
        full = torch.full((B,), ctx, dtype=torch.int32, device=dev)
        ones = np.ones(B, dtype=np.int32)
        batch = StepBatch(num_tokens=B, num_requests=B, num_logit_rows=B, max_q_len=1, max_kv_len=ctx + 1,
                          token_ids=torch.zeros(B, dtype=torch.int32, device=dev), positions=full, tok_req=ar[:B],
                          q_start=ar, pos_start=full, kv_len=full + 1, slots=ar[:B], logit_rows=ar[:B], req_order=ar[:B],
                          block_tables=[table], h_q_lens=ones, h_pos_start=ones * ctx, h_sorted_q_lens=ones,
                          h_sorted_kv_lens=ones * (ctx + 1), all_decode=True, real_requests=B, real_logit_rows=B)
        byts = B * (ctx + 1) * 2 * nkv * d * 2

        def call():
            ops.attention_bf16(q, batch, table, cache, 0, page, out, nq, nkv, d, 1 / math.sqrt(d), 0)
        for _ in range(3):
            call()
        times = []
        for _ in range(iters):
            flush.zero_()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            call()
            b.record()
            torch.cuda.synchronize()
            times.append(a.elapsed_time(b) * 1e3)
        ops.check_errors()
        us = statistics.median(times)
        print(json.dumps({"point": "attn_decode", "requests": B, "context": ctx, "mbytes": round(byts / 1e6, 1),
                          "us": round(us, 1), "us_at_copy_rate": round(byts / peaks["hbm_gbs"] / 1e3, 1),
                          "key_shares": ops.attention_splits(B, 1, nq, nkv), "peaks": peaks["source"]}), flush=True)
        del cache
    return 0


# ------------------------------------------------------------------ the Tipezen design beside Qwen3 at equal layer sizes
# (width, query heads, key/value heads, head size, feed-forward, window, retention heads) of two sizes that resemble a
# real model's layers; the Tipezen model alternates retention layers without a feed-forward and attention layers with
# one, over four residual streams; its twin is Qwen3 with as many layers of the same width, heads and feed-forward.
TIPEZEN_SIZES = {"2k": (2048, 16, 4, 128, 6144, 1024, 16), "4k": (4096, 32, 8, 128, 12288, 2048, 32)}
TIPEZEN_LAYERS = 8
TIPEZEN_VOCAB = 32768


def tipezen_engine(size: str, max_live: int, cache_tokens: int, graphs: bool, step_tokens: int):
    import torch
    import tffinfer_b200 as tff
    from tffinfer_b200.config import TipezenConfig, TipezenLayer, RotaryConfig
    from tffinfer_b200.weights import random_tensors_on_device
    W, H, G, D, F, win, RH = TIPEZEN_SIZES[size]
    att = TipezenLayer(type="attention", heads=H, kv_heads=G, dim=D, vdim=D, scale=D ** -0.5, softcap=50.0, window=win,
                       v_mix=True, rot=RotaryConfig(5e4, D, (4.0, 4096.0, 16.0, 1.0)), ff=F)
    ret = TipezenLayer(type="retention", heads=RH, dim=D, vdim=D, rot=RotaryConfig(5e5, D),
                       decay=tuple(1.0 - 2.0 ** (-5 - 4 * i / RH) for i in range(RH)))
    cfg = TipezenConfig("Tipezen", vocab_size=TIPEZEN_VOCAB, hidden_size=W, streams=4, norm_eps=1e-6,
                        layers=tuple(ret if i % 2 == 0 else att for i in range(TIPEZEN_LAYERS)))
    tensors = random_tensors_on_device(cfg, 0, "cuda", "bfloat16")
    ecfg = tff.EngineConfig(dtype="bfloat16", page_size=PAGE_SIZE, max_cache_tokens=cache_tokens, max_live_requests=max_live,
                            max_tokens_per_step=step_tokens, max_model_len=8192, use_cuda_graphs=graphs)
    runner = tff.ModelRunner(config=cfg, tensors=tensors, engine_config=ecfg)
    del tensors
    torch.cuda.empty_cache()
    return tff.Engine(runner=runner), cfg


def qwen_twin_engine(size: str, max_live: int, cache_tokens: int, graphs: bool, step_tokens: int):
    import torch
    import tffinfer_b200 as tff
    from tffinfer_b200.config import Qwen3Config
    from tffinfer_b200.weights import random_tensors_on_device
    W, H, G, D, F, win, _ = TIPEZEN_SIZES[size]
    cfg = Qwen3Config(architecture="Qwen3ForCausalLM", hidden_size=W, num_layers=TIPEZEN_LAYERS, num_heads=H, num_kv_heads=G,
                      head_dim=D, intermediate_size=F, vocab_size=TIPEZEN_VOCAB, rms_norm_eps=1e-6, rope_theta=1e6,
                      max_position=8192, tie_word_embeddings=False, sliding_window=win,
                      layer_types=tuple("sliding_attention" if i % 2 else "full_attention" for i in range(TIPEZEN_LAYERS))).validate()
    tensors = random_tensors_on_device(cfg, 0, "cuda", "bfloat16")
    ecfg = tff.EngineConfig(dtype="bfloat16", page_size=PAGE_SIZE, max_cache_tokens=cache_tokens, max_live_requests=max_live,
                            max_tokens_per_step=step_tokens, max_model_len=8192, use_cuda_graphs=graphs)
    runner = tff.ModelRunner(config=cfg, tensors=tensors, engine_config=ecfg)
    del tensors
    torch.cuda.empty_cache()
    return tff.Engine(runner=runner), cfg


def traced_kinds(engine, prompt_len: int, batch: int):
    """Device time by kind of kernel call of one whole-prompt step and of one decode step of ``batch`` requests
    behind such prompts, launched kernel by kernel (the engine was made without CUDA graphs)."""
    import torch
    from tffinfer_b200 import StepEntry
    from tffinfer_b200.kernels.trace import KernelTrace
    runner = engine.runner
    rng = random.Random(3)
    vocab = runner.desc.vocab_size
    ids = [f"t{i}" for i in range(batch)]
    for rid in ids:
        runner.add_request(rid)
    prompt = lambda: [rng.randrange(vocab) for _ in range(prompt_len)]
    out = {}
    runner.step([StepEntry(ids[0], prompt(), [prompt_len - 1])])            # every prompt-sized kernel has run once
    torch.cuda.synchronize()
    with KernelTrace(runner.ops) as tr:
        runner.step([StepEntry(ids[1], prompt(), [prompt_len - 1])])
    out["prefill"] = {k: (c, round(ms, 4)) for k, c, ms in tr.summary()}
    for rid in ids[2:]:
        runner.step([StepEntry(rid, prompt(), [])])
    runner.step([StepEntry(rid, [1], [0]) for rid in ids])                   # and every decode-sized one
    torch.cuda.synchronize()
    with KernelTrace(runner.ops) as tr:
        runner.step([StepEntry(rid, [(7919 * i + 2) % vocab], [0]) for i, rid in enumerate(ids)])
    out["decode"] = {k: (c, round(ms, 4)) for k, c, ms in tr.summary()}
    for rid in ids:
        runner.finish_request(rid)
    return out


def run_tipezen(steps: int, warmup: int) -> int:
    """Prefill and decode throughput of the Tipezen design at two layer sizes beside Qwen3 at the same sizes, one JSON
    line a point, and for each model the device time of a step by kind of kernel call with what the new kernels
    reach of the measured copy rate (streams, rotation and cache write, decode retention) or of the float32 FMA
    rate of the device (chunked retention)."""
    import torch
    peaks = load_peaks()
    steps = min(steps, 32)
    P = PROMPT_LEN
    for size in TIPEZEN_SIZES:
        W, H, G, D, F, win, RH = TIPEZEN_SIZES[size]
        for model, make in (("tipezen", tipezen_engine), ("qwen3", qwen_twin_engine)):
            need = 64 * (P + warmup + steps + 64 + 72)
            engine, cfg = make(size, 64, need, True, P)
            pms = prefill_run(engine, iters=3, warmup=2, seed=1, prompt_len=P)
            print(json.dumps({"point": "prefill", "model": model, "size": size, "layers": TIPEZEN_LAYERS, "tokens": P,
                              "ms": round(pms, 3), "tok_s": round(P / (pms / 1e3), 1)}), flush=True)
            for b in (8, 64):
                run = decode_run(engine, b, steps, warmup, seed=b, prompt_len=P)
                print(json.dumps({"point": "decode", "model": model, "size": size, "layers": TIPEZEN_LAYERS, "batch": b,
                                  "context": round(run["mean_context"]), "tok_s": round(run["tok_s"], 1),
                                  "ms_per_step": round(run["ms_per_step"], 4), "launches_per_step": run["launches"] // steps}),
                      flush=True)
            del engine
            torch.cuda.empty_cache()
            engine, cfg = make(size, 8, 8 * (P + 64), False, P)
            kinds = traced_kinds(engine, P, 8)
            line = {"point": "kernels", "model": model, "size": size, "prefill_tokens": P, "decode_batch": 8,
                    "prefill_ms_by_kind": kinds.get("prefill"), "decode_ms_by_kind": kinds.get("decode"), "peaks": peaks["source"]}
            if model == "tipezen":
                nl = TIPEZEN_LAYERS // 2
                S = 4
                # bytes a call must move, summed over the step's calls of the kind
                subl = nl * 3                                  # sublayers: a mixer a layer, a feed-forward every other
                stream_b = lambda T: (subl + 1) * T * (2 * S * W * 4 + W * 4 + W * 2)
                finish_b = lambda T: nl * T * ((2 * RH * D + 2 * RH * D) * 4 + (2 * RH * D) * 4) + \
                    nl * T * ((H + 2 * G) * D * 4 + H * D * 2 + 2 * G * D * 2 + 2 * G * D * 4)
                state_b = nl * 8 * RH * D * D * 4 * 2          # decode: every request's state read and written
                # chunks of 64 tokens: A = Q K^T and A V (64 x 64 x D each), U = K^T V and Q S (64 x D x D each)
                ret_flops = lambda T: nl * RH * (T / 64.0) * 2.0 * 64 * D * (2 * 64 + 2 * D)
                fr = {}
                for step, T in (("prefill", P), ("decode", 8)):
                    k = kinds.get(step) or {}
                    if "stream_step" in k:
                        fr[f"{step}_stream_step_hbm_frac"] = round(stream_b(T) / (k["stream_step"][1] / 1e3) / 1e9 / peaks["hbm_gbs"], 4)
                    if "qkv_finish" in k:
                        fr[f"{step}_qkv_finish_hbm_frac"] = round(finish_b(T) / (k["qkv_finish"][1] / 1e3) / 1e9 / peaks["hbm_gbs"], 4)
                if "retention" in (kinds.get("decode") or {}):
                    fr["decode_retention_hbm_frac"] = round(state_b / (kinds["decode"]["retention"][1] / 1e3) / 1e9 / peaks["hbm_gbs"], 4)
                if "retention" in (kinds.get("prefill") or {}):
                    fr["prefill_retention_fp32_tflops"] = round(ret_flops(P) / (kinds["prefill"]["retention"][1] / 1e3) / 1e12, 2)
                line["fractions"] = fr
            print(json.dumps(line), flush=True)
            del engine
            torch.cuda.empty_cache()
    return 0

# The Dominex design beside Tipezen (the closest of the other models: layers listed one by one, a windowed attention
# beside a recurrence with state slots) at the same width: (width, latent heads, dim, rot_dim, vdim, q_rank, kv_rank,
# left heads, left kv heads, left dim, block, recurrence width, experts, chosen, expert ff).  Four layers of two mixers
# side by side alternate with four latent attention layers (one of them reading its neighbour's vectors); the latent
# layers carry the experts, whose chosen share equals the twin's dense feed-forward.
DOMINEX_SIZES = {"2k": (2048, 16, 128, 64, 128, 768, 512, 16, 4, 128, 1024, 2048, 16, 2, 3072),
                 "4k": (4096, 32, 128, 64, 128, 1536, 512, 32, 8, 128, 2048, 4096, 16, 2, 6144)}


def dominex_engine(size: str, max_live: int, cache_tokens: int, graphs: bool, step_tokens: int):
    import torch
    import tffinfer_b200 as tff
    from tffinfer_b200.config import DominexConfig, DominexLayer, DominexExperts
    from tffinfer_b200.weights import random_tensors_on_device
    W, H, D, R, VD, QR, KR, LH, LG, LD, CH, RW, E, TOP, F = DOMINEX_SIZES[size]
    moe = DominexExperts(ff=F, experts=E, top=TOP)
    lat = lambda src: DominexLayer(type="latent_attention", heads=H, dim=D, rot_dim=R, vdim=VD, q_rank=QR, kv_rank=KR,
                                   scale=(D + R) ** -0.5, rot_base=5e5, rot_dims=R, kv_from=src, mlp=moe)
    par = DominexLayer(type="parallel", left_heads=LH, left_kv_heads=LG, left_dim=LD, left_vdim=LD, left_scale_qk=LD ** -0.5,
                       left_chunk=CH, right_width=RW, left_scale=0.8, right_scale=0.9)
    layers = tuple(par if i % 2 == 0 else lat(1 if i == 5 else None) for i in range(TIPEZEN_LAYERS))
    cfg = DominexConfig("Dominex", vocab_size=TIPEZEN_VOCAB, hidden_size=W, embed_scale=W ** 0.5, norm_eps=1e-6,
                        logit_softcap=30.0, layers=layers)
    tensors = random_tensors_on_device(cfg, 0, "cuda", "bfloat16")
    ecfg = tff.EngineConfig(dtype="bfloat16", page_size=PAGE_SIZE, max_cache_tokens=cache_tokens, max_live_requests=max_live,
                            max_tokens_per_step=step_tokens, max_model_len=8192, use_cuda_graphs=graphs)
    runner = tff.ModelRunner(config=cfg, tensors=tensors, engine_config=ecfg)
    del tensors
    torch.cuda.empty_cache()
    return tff.Engine(runner=runner), cfg


def run_dominex(steps: int, warmup: int, sizes=None) -> int:
    """Prefill and decode throughput of the Dominex design beside Tipezen at the same layer sizes, one JSON line a
    point, and for each model the device time of a step by kind of kernel call; for Dominex also what its own
    kernels reach: the attention tiles and the grouped products in TFLOP/s, the recurrence and the small kernels
    around the experts as a fraction of the measured copy rate."""
    import torch
    peaks = load_peaks()
    steps = min(steps, 32)
    P = PROMPT_LEN
    for size in (sizes or DOMINEX_SIZES):
        W, H, D, R, VD, QR, KR, LH, LG, LD, CH, RW, E, TOP, F = DOMINEX_SIZES[size]
        for model, make in (("dominex", dominex_engine), ("tipezen", tipezen_engine)):
            need = 64 * (P + warmup + steps + 64 + 72)
            engine, cfg = make(size, 64, need, True, P)
            pms = prefill_run(engine, iters=3, warmup=2, seed=1, prompt_len=P)
            print(json.dumps({"point": "prefill", "model": model, "size": size, "layers": TIPEZEN_LAYERS, "tokens": P,
                              "ms": round(pms, 3), "tok_s": round(P / (pms / 1e3), 1)}), flush=True)
            for b in (8, 64):
                run = decode_run(engine, b, steps, warmup, seed=b, prompt_len=P)
                print(json.dumps({"point": "decode", "model": model, "size": size, "layers": TIPEZEN_LAYERS, "batch": b,
                                  "context": round(run["mean_context"]), "tok_s": round(run["tok_s"], 1),
                                  "ms_per_step": round(run["ms_per_step"], 4), "launches_per_step": run["launches"] // steps}),
                      flush=True)
            del engine
            torch.cuda.empty_cache()
            engine, cfg = make(size, 8, 8 * (P + 64), False, P)
            kinds = traced_kinds(engine, P, 8)
            line = {"point": "kernels", "model": model, "size": size, "prefill_tokens": P, "decode_batch": 8,
                    "prefill_ms_by_kind": kinds.get("prefill"), "decode_ms_by_kind": kinds.get("decode"), "peaks": peaks["source"]}
            if model == "dominex":
                nl = TIPEZEN_LAYERS // 2
                # prompt step: causal scores and weighted sums of the latent layers (keys of KR + R, values of KR
                # elements, H heads) and of the chunked layers (LD and LD, LH heads, blocks of CH positions)
                pairs = lambda T, span: T * (min(T, span) + 1) / 2.0 if span >= T else T * (span + 1) / 2.0
                # (whole prompts: the latent layers make per-head keys of D + R and values of VD elements for the step's tokens)
                attn_flops = nl * H * pairs(P, P) * 2.0 * (D + R + VD) + nl * LH * pairs(P, CH) * 2.0 * (2 * LD)
                expert_flops = nl * P * TOP * 3 * 2.0 * W * F
                head_flops = nl * P * H * 2.0 * KR * (D + VD)
                gru_bytes = lambda T: nl * T * RW * (3 * 4 + 2)
                fr = {}
                k = kinds.get("prefill") or {}
                if "attention_tile" in k:
                    fr["prefill_attention_tile_tflops"] = round(attn_flops / (k["attention_tile"][1] / 1e3) / 1e12, 2)
                if "gemm_tc_grouped" in k:
                    fr["prefill_experts_tcgen05_tflops"] = round(expert_flops / (k["gemm_tc_grouped"][1] / 1e3) / 1e12, 2)
                    fr["prefill_experts_tcgen05_frac"] = round(fr["prefill_experts_tcgen05_tflops"] / peaks["bf16_tflops"], 4)
                if "gemm_grouped" in k:
                    flops = head_flops if "gemm_tc_grouped" in k else head_flops + expert_flops
                    fr["prefill_gemm_grouped_tflops"] = round(flops / (k["gemm_grouped"][1] / 1e3) / 1e12, 2)
                if "min_gru" in k:
                    fr["prefill_min_gru_hbm_frac"] = round(gru_bytes(P) / (k["min_gru"][1] / 1e3) / 1e9 / peaks["hbm_gbs"], 4)
                kd = kinds.get("decode") or {}
                if "attention_tile" in kd:
                    # decode: every request's cached vectors (latent) and the keys and values of its block are read once
                    cache_b = 8 * (3 * P * (KR + R) * 2 + nl * min(P, CH) * 2 * LG * LD * 2)
                    fr["decode_attention_tile_hbm_frac"] = round(cache_b / (kd["attention_tile"][1] / 1e3) / 1e9 / peaks["hbm_gbs"], 4)
                if "gemm_grouped" in kd:
                    # decode: the chosen experts' weights (at most 8 * TOP different ones of E) and the heads' up-projections
                    w_b = nl * (min(E, 8 * TOP) * 3 * W * F * 2 + H * KR * (D + VD) * 2)
                    fr["decode_gemm_grouped_hbm_frac"] = round(w_b / (kd["gemm_grouped"][1] / 1e3) / 1e9 / peaks["hbm_gbs"], 4)
                line["fractions"] = fr
            print(json.dumps(line), flush=True)
            del engine
            torch.cuda.empty_cache()
    return 0


# The Sadupel design beside Dominex (the closest of the other models: layers listed one by one, routed experts behind a
# softmax attention over the paged cache) at the same width: (width, heads, kv heads, dim, taps, experts, identity
# experts, chosen, groups, kept groups, expert ff, shared ff).  Six layers, of which layers 2 and 3 run twice in a row
# (eight layer runs, as many as the twin has layers); the experts are not gated, so their ff is 1.5 times the twin's for
# the same arithmetic a chosen expert.
SADUPEL_SIZES = {"2k": (2048, 16, 4, 128, 4, 14, 2, 2, 4, 2, 4608, 2048),
                 "4k": (4096, 32, 8, 128, 4, 14, 2, 2, 4, 2, 9216, 4096)}
SADUPEL_RUNS = 8


def sadupel_engine(size: str, max_live: int, cache_tokens: int, graphs: bool, step_tokens: int):
    import torch
    import tffinfer_b200 as tff
    from tffinfer_b200.config.sadupel_config import SadupelConfig, SadupelLayer, SadupelExperts
    from tffinfer_b200.weights import random_tensors_on_device
    W, H, G, D, TAPS, E, IDENT, TOP, GROUPS, KEEP, F, SF = SADUPEL_SIZES[size]
    moe = SadupelExperts(ff=F, experts=E, top=TOP, identity=IDENT, groups=GROUPS, keep=KEEP, shared_ff=SF)
    layer = SadupelLayer(heads=H, kv_heads=G, dim=D, vdim=D, conv=TAPS, scale=D ** -0.5, softcap=30.0, rot_base=5e5,
                         rot_dims=D // 2, rot_factor=4.0, mlp=moe)
    cfg = SadupelConfig("Sadupel", vocab_size=TIPEZEN_VOCAB, hidden_size=W, norm_eps=1e-6, residual_mult=0.5,
                        bigram=(65521, 31, 17), loop=(2, 4, 2), layers=(layer,) * 6)
    assert len(cfg.runs()) == SADUPEL_RUNS
    tensors = random_tensors_on_device(cfg, 0, "cuda", "bfloat16")
    ecfg = tff.EngineConfig(dtype="bfloat16", page_size=PAGE_SIZE, max_cache_tokens=cache_tokens, max_live_requests=max_live,
                            max_tokens_per_step=step_tokens, max_model_len=8192, use_cuda_graphs=graphs)
    runner = tff.ModelRunner(config=cfg, tensors=tensors, engine_config=ecfg)
    del tensors
    torch.cuda.empty_cache()
    return tff.Engine(runner=runner), cfg


def run_sadupel(steps: int, warmup: int, sizes=None) -> int:
    """Prefill and decode throughput of the Sadupel design beside Dominex at the same layer sizes, one JSON line a
    point, and for each model the device time of a step by kind of kernel call; for Sadupel also what its own kernels
    reach: the convolution-and-norm kernel, the hashed embedding, the router and the activation kernels as a fraction of
    the measured copy rate, the attention and the experts' grouped products in TFLOP/s."""
    import torch
    peaks = load_peaks()
    steps = min(steps, 32)
    P = PROMPT_LEN
    clocks = ClockSampler()            # over the whole run: SM clock at the median, the throttle reasons seen
    clocks.start()
    for size in (sizes or SADUPEL_SIZES):
        W, H, G, D, TAPS, E, IDENT, TOP, GROUPS, KEEP, F, SF = SADUPEL_SIZES[size]
        for model, make in (("sadupel", sadupel_engine), ("dominex", dominex_engine)):
            need = 64 * (P + warmup + steps + 64 + 72)
            engine, cfg = make(size, 64, need, True, P)
            pms = prefill_run(engine, iters=3, warmup=2, seed=1, prompt_len=P)
            print(json.dumps({"point": "prefill", "model": model, "size": size, "layers": TIPEZEN_LAYERS, "tokens": P,
                              "ms": round(pms, 3), "tok_s": round(P / (pms / 1e3), 1)}), flush=True)
            for b in (8, 64):
                run = decode_run(engine, b, steps, warmup, seed=b, prompt_len=P)
                print(json.dumps({"point": "decode", "model": model, "size": size, "layers": TIPEZEN_LAYERS, "batch": b,
                                  "context": round(run["mean_context"]), "tok_s": round(run["tok_s"], 1),
                                  "ms_per_step": round(run["ms_per_step"], 4), "launches_per_step": run["launches"] // steps}),
                      flush=True)
            del engine
            torch.cuda.empty_cache()
            engine, cfg = make(size, 8, 8 * (P + 64), False, P)
            kinds = traced_kinds(engine, P, 8)
            line = {"point": "kernels", "model": model, "size": size, "prefill_tokens": P, "decode_batch": 8,
                    "prefill_ms_by_kind": kinds.get("prefill"), "decode_ms_by_kind": kinds.get("decode"), "peaks": peaks["source"]}
            if model == "sadupel":
                nl = SADUPEL_RUNS
                C = (H + 2 * G) * D                       # channels of q, k and v together
                ld = -(-(C + H) // 8) * 8                 # with the head gates, padded
                # convolution and norm: a row of float32 accumulators read and a float32 row written (the taps' older rows
                # come from the cache of the chip); the state kernel reads the last rows again and clears nothing here
                conv_b = lambda T: nl * T * ld * 4 * 2
                finish_b = lambda T: nl * T * (ld * 4 + H * D * 2 + 2 * G * D * 2 + H * 4)
                # the share of chosen outputs that are experts with rows is not known ahead: all TOP are counted
                expert_flops = nl * P * TOP * 2 * 2.0 * W * F
                attn_flops = nl * H * (P * (P + 1) / 2.0) * 2.0 * (2 * D)
                fr = {}
                for step, T in (("prefill", P), ("decode", 8)):
                    k = kinds.get(step) or {}
                    if "short_conv_norm" in k:
                        fr[f"{step}_short_conv_norm_hbm_frac"] = round(conv_b(T) / (k["short_conv_norm"][1] / 1e3) / 1e9 / peaks["hbm_gbs"], 4)
                    if "qkv_finish" in k:
                        fr[f"{step}_qkv_finish_hbm_frac"] = round(finish_b(T) / (k["qkv_finish"][1] / 1e3) / 1e9 / peaks["hbm_gbs"], 4)
                k = kinds.get("prefill") or {}
                if "gemm_tc_grouped" in k:
                    fr["prefill_experts_tcgen05_tflops"] = round(expert_flops / (k["gemm_tc_grouped"][1] / 1e3) / 1e12, 2)
                    fr["prefill_experts_tcgen05_frac"] = round(fr["prefill_experts_tcgen05_tflops"] / peaks["bf16_tflops"], 4)
                if "attention_bf16" in k:
                    fr["prefill_attention_tflops"] = round(attn_flops / (k["attention_bf16"][1] / 1e3) / 1e12, 2)
                kd = kinds.get("decode") or {}
                if "gemm_grouped" in kd:
                    # the experts a step of 8 tokens touches: with random weights every choice is one of E + IDENT outputs,
                    # so of the E experts with tensors about E * (1 - (1 - TOP / outputs)^8) are read
                    touched = E * (1.0 - (1.0 - TOP / float(E + IDENT)) ** 8)
                    w_b = nl * touched * 2 * W * F * 2
                    fr["decode_experts_touched"] = round(touched, 1)
                    fr["decode_gemm_grouped_hbm_frac"] = round(w_b / (kd["gemm_grouped"][1] / 1e3) / 1e9 / peaks["hbm_gbs"], 4)
                if "attention_bf16" in kd:
                    cache_b = nl * 8 * P * 2 * G * D * 2
                    fr["decode_attention_hbm_frac"] = round(cache_b / (kd["attention_bf16"][1] / 1e3) / 1e9 / peaks["hbm_gbs"], 4)
                line["fractions"] = fr
            print(json.dumps(line), flush=True)
            del engine
            torch.cuda.empty_cache()
    clocks.stop()
    print(json.dumps({"point": "clocks", "clocks": clocks.summary()}), flush=True)
    return 0


# The Nugosun design beside Dominex (the closest of the other models: layers listed one by one, a chunked attention
# beside a recurrence with state slots, latent attention with borrowed vectors, routed experts) at the same width:
# (width, latent heads, dim, rot_dim, vdim, q_rank, kv_rank, left heads, left kv heads, left dim, block, state-space heads,
# head channels, state rows, gla heads, gla key size, gla value size, experts, chosen, expert ff, dense ff).  Eight layers:
# parallel, latent, gla, gla, parallel, latent (reading layer 1's vectors), gla, latent; dense and routed feed-forwards
# take turns.
NUGOSUN_SIZES = {"2k": (2048, 16, 128, 64, 128, 768, 512, 16, 4, 128, 1024, 32, 64, 128, 8, 128, 256, 16, 2, 3072, 6144),
                 "4k": (4096, 32, 128, 64, 128, 1536, 512, 32, 8, 128, 2048, 64, 64, 128, 16, 128, 256, 16, 2, 6144, 12288)}
NUGOSUN_ORDER = ("parallel", "latent", "gla", "gla", "parallel", "latent", "gla", "latent")


def nugosun_engine(size: str, max_live: int, cache_tokens: int, graphs: bool, step_tokens: int):
    import torch
    import tffinfer_b200 as tff
    from tffinfer_b200.config.nugosun_config import (NugosunConfig, NugosunLayer, NugosunMlp, NugosunGla, NugosunAttention,
                                                     NugosunStateSpace, NugosunLatent)
    from tffinfer_b200.config.tipezen_config import RotaryConfig
    from tffinfer_b200.weights import random_tensors_on_device
    W, H, D, R, VD, QR, KR, LH, LG, LD, CH, SH, SP, SN, GH, GK, GV, E, TOP, F, DF = NUGOSUN_SIZES[size]
    moe, dense = NugosunMlp("moe", F, E, TOP), NugosunMlp("dense", DF)
    layers = []
    for i, kind in enumerate(NUGOSUN_ORDER):
        mlp = moe if i % 2 else dense
        if kind == "parallel":
            layers.append(NugosunLayer("parallel", left=NugosunAttention(
                LH, LG, LD, LD, LD ** -0.5 * 4.0, 30.0, CH, RotaryConfig(1e6, LD // 2, (4.0, 4096.0, 16.0, 2.0))),
                right=NugosunStateSpace(SH, SP, SN, 1, 4, 1), left_scale=0.8, right_scale=0.9, mlp=mlp))
        elif kind == "latent":
            layers.append(NugosunLayer("latent_attention", latent=NugosunLatent(
                H, D, R, VD, QR, KR, (D + R) ** -0.5, RotaryConfig(5e5, R), 1 if i == 5 else None), mlp=mlp))
        else:
            layers.append(NugosunLayer("gla", gla=NugosunGla(GH, GK, GV, 16.0, 16), mlp=mlp))
    cfg = NugosunConfig("Nugosun", vocab_size=TIPEZEN_VOCAB, hidden_size=W, embed_scale=W ** 0.5, norm_eps=1e-6,
                        layers=tuple(layers))
    tensors = random_tensors_on_device(cfg, 0, "cuda", "bfloat16")
    ecfg = tff.EngineConfig(dtype="bfloat16", page_size=PAGE_SIZE, max_cache_tokens=cache_tokens, max_live_requests=max_live,
                            max_tokens_per_step=step_tokens, max_model_len=8192, use_cuda_graphs=graphs)
    runner = tff.ModelRunner(config=cfg, tensors=tensors, engine_config=ecfg)
    del tensors
    torch.cuda.empty_cache()
    return tff.Engine(runner=runner), cfg


def run_nugosun(steps: int, warmup: int, sizes=None) -> int:
    """Prefill and decode throughput of the Nugosun design beside Dominex at the same layer sizes, one JSON line a point,
    and for each model the device time of a step by kind of kernel call; for Nugosun also what its own kernels reach
    as a fraction of the measured copy rate: the recurrence over the matrix states (the rows it reads and writes in a
    prompt step, the states it reads and writes in a decode step), the convolution, the gated norm, the two norms in one
    pass, and the rotation-and-cache-write kernel with biases and unit-norm heads."""
    import torch
    peaks = load_peaks()
    steps = min(steps, 32)
    P = PROMPT_LEN
    clocks = ClockSampler()
    clocks.start()
    for size in (sizes or NUGOSUN_SIZES):
        W, H, D, R, VD, QR, KR, LH, LG, LD, CH, SH, SP, SN, GH, GK, GV, E, TOP, F, DF = NUGOSUN_SIZES[size]
        for model, make in (("nugosun", nugosun_engine), ("dominex", dominex_engine)):
            need = 64 * (P + warmup + steps + 64 + 72)
            engine, cfg = make(size, 64, need, True, P)
            pms = prefill_run(engine, iters=3, warmup=2, seed=1, prompt_len=P)
            print(json.dumps({"point": "prefill", "model": model, "size": size, "layers": TIPEZEN_LAYERS, "tokens": P,
                              "ms": round(pms, 3), "tok_s": round(P / (pms / 1e3), 1)}), flush=True)
            for b in (8, 64):
                run = decode_run(engine, b, steps, warmup, seed=b, prompt_len=P)
                print(json.dumps({"point": "decode", "model": model, "size": size, "layers": TIPEZEN_LAYERS, "batch": b,
                                  "context": round(run["mean_context"]), "tok_s": round(run["tok_s"], 1),
                                  "ms_per_step": round(run["ms_per_step"], 4), "launches_per_step": run["launches"] // steps}),
                      flush=True)
            del engine
            torch.cuda.empty_cache()
            engine, cfg = make(size, 8, 8 * (P + 64), False, P)
            kinds = traced_kinds(engine, P, 8)
            line = {"point": "kernels", "model": model, "size": size, "prefill_tokens": P, "decode_batch": 8,
                    "prefill_ms_by_kind": kinds.get("prefill"), "decode_ms_by_kind": kinds.get("decode"), "peaks": peaks["source"]}
            if model == "nugosun":
                n_par, n_gla, n_lay = NUGOSUN_ORDER.count("parallel"), NUGOSUN_ORDER.count("gla"), len(NUGOSUN_ORDER)
                inner, ch = SH * SP, SH * SP + 2 * SN
                # the recurrence: float32 rows read (q, k, decay, v) and written (o) a token; a request's states read and written a step
                rec_rows = lambda T: 4 * T * (n_gla * (3 * GH * GK + 2 * GH * GV) + n_par * (2 * SN + SH + 2 * inner))
                rec_state = lambda B: 4 * 2 * B * (n_gla * GH * GK * GV + n_par * SH * SN * SP)
                conv_b = lambda T: n_par * T * ch * 4 * 2
                gnorm_b = lambda T: n_gla * T * GH * GV * (4 + 4 + 2) + n_par * T * inner * (4 + 4 + 2)
                pair_b = lambda T: n_lay * T * W * (4 + 2 + 2)
                finish_b = lambda T: n_par * T * ((LH + 2 * LG) * LD * 4 + LH * LD * 2 + 2 * LG * LD * 2)
                fr = {}
                for step, T, B in (("prefill", P, 1), ("decode", 8, 8)):
                    k = kinds.get(step) or {}
                    for kind, nbytes in (("linear_recurrence", rec_rows(T) + rec_state(B)), ("causal_conv", conv_b(T)),
                                         ("gated_norm", gnorm_b(T)), ("rmsnorm_pair", pair_b(T)), ("qkv_finish", finish_b(T))):
                        if kind in k:
                            fr[f"{step}_{kind}_hbm_frac"] = round(nbytes / (k[kind][1] / 1e3) / 1e9 / peaks["hbm_gbs"], 4)
                k = kinds.get("prefill") or {}
                if "linear_recurrence" in k:      # multiply-adds of the recurrence: decay, outer product and read-out a state element
                    flops = P * 6.0 * (n_gla * GH * GK * GV + n_par * SH * SN * SP)
                    fr["prefill_linear_recurrence_fp32_tflops"] = round(flops / (k["linear_recurrence"][1] / 1e3) / 1e12, 2)
                line["fractions"] = fr
            print(json.dumps(line), flush=True)
            del engine
            torch.cuda.empty_cache()
    clocks.stop()
    print(json.dumps({"point": "clocks", "clocks": clocks.summary()}), flush=True)
    return 0


# The Kadodra design beside Nugosun (the closest of the other models: latent attention and linear attention over matrix
# states, two sublayers side by side, dense and routed feed-forwards) at the same width: (width, latent heads, dim, rot_dim,
# vdim, kv_rank, window, lightning heads, key size, value size, experts, chosen, expert ff, dense ff).  Six layers, lightning
# and latent in turn, of which layers 2 and 3 run twice (eight layer runs, as many as the twin has layers); the dense
# feed-forward has no gate, so its ff is 1.5 times the twin's for the same arithmetic.
KADODRA_SIZES = {"2k": (2048, 16, 128, 64, 128, 512, 1024, 16, 128, 128, 16, 2, 3072, 9216),
                 "4k": (4096, 32, 128, 64, 128, 512, 1024, 32, 128, 128, 16, 2, 6144, 18432)}
KADODRA_LOOP = (2, 4, 2)


def kadodra_engine(size: str, max_live: int, cache_tokens: int, graphs: bool, step_tokens: int):
    import torch
    import tffinfer_b200 as tff
    from tffinfer_b200.config.kadodra_config import KadodraConfig, KadodraLayer, KadodraMlp, KadodraLatent, KadodraLightning
    from tffinfer_b200.config.tipezen_config import RotaryConfig
    from tffinfer_b200.weights import random_tensors_on_device
    W, H, D, R, VD, KR, WIN, LH, LD, LV, E, TOP, F, DF = KADODRA_SIZES[size]
    light = KadodraLayer("lightning", mlp=KadodraMlp("dense", DF), lightning=KadodraLightning(
        LH, LD, LV, tuple(1.0 - 2.0 ** -(3 + 6.0 * i / LH) for i in range(LH))))
    latent = KadodraLayer("latent_attention", mlp=KadodraMlp("moe", F, E, TOP, 7.0), latent=KadodraLatent(
        H, D, R, VD, KR, (D + R) ** -0.5, RotaryConfig(5e5, R, (4.0, 4096.0, 16.0, 2.0)), WIN))
    cfg = KadodraConfig("Kadodra", vocab_size=TIPEZEN_VOCAB, hidden_size=W, norm_eps=1e-6, logit_scale=0.25, loop=KADODRA_LOOP,
                        layers=(light, latent) * 3)
    tensors = random_tensors_on_device(cfg, 0, "cuda", "bfloat16")
    ecfg = tff.EngineConfig(dtype="bfloat16", page_size=PAGE_SIZE, max_cache_tokens=cache_tokens, max_live_requests=max_live,
                            max_tokens_per_step=step_tokens, max_model_len=8192, use_cuda_graphs=graphs)
    runner = tff.ModelRunner(config=cfg, tensors=tensors, engine_config=ecfg)
    del tensors
    torch.cuda.empty_cache()
    return tff.Engine(runner=runner), cfg


def experts_of(engine, tokens):
    """{"experts_touched": how many experts of a layer a step of these tokens reads, on average over the layers} where a
    table of token ids chooses the experts; {} for other models."""
    tables = [b.feed_forward.table for b in engine.runner.model.blocks if getattr(b.feed_forward, "table", None) is not None]
    if not tables:
        return {}
    return {"experts_touched": round(sum(len(set(t[list(tokens)].flatten().tolist())) for t in tables) / len(tables), 1)}


def run_kadodra(steps: int, warmup: int, sizes=None) -> int:
    """Prefill and decode throughput of the Kadodra design beside Nugosun at the same layer sizes, one JSON line a point,
    and for each model the device time of a step by kind of kernel call; for Kadodra also what its own kernels reach: the
    recurrence in TFLOP/s of its chunk form (prompt step) and as a fraction of the measured copy rate for the states it
    reads and writes (decode step), the norm over all heads, the kernel between the latent projections and the attention,
    the sorting by the table and the sum of experts as fractions of the copy rate, the windowed attention and the experts'
    products in TFLOP/s."""
    import torch
    peaks = load_peaks()
    steps = min(steps, 32)
    P = PROMPT_LEN
    clocks = ClockSampler()
    clocks.start()
    for size in (sizes or KADODRA_SIZES):
        W, H, D, R, VD, KR, WIN, LH, LD, LV, E, TOP, F, DF = KADODRA_SIZES[size]
        for model, make in (("kadodra", kadodra_engine), ("nugosun", nugosun_engine)):
            need = 64 * (P + warmup + steps + 64 + 72)
            engine, cfg = make(size, 64, need, True, P)
            pms = prefill_run(engine, iters=3, warmup=2, seed=1, prompt_len=P)
            print(json.dumps({"point": "prefill", "model": model, "size": size, "layers": TIPEZEN_LAYERS, "tokens": P,
                              "ms": round(pms, 3), "tok_s": round(P / (pms / 1e3), 1)}), flush=True)
            for b in (8, 64):
                run = decode_run(engine, b, steps, warmup, seed=b, prompt_len=P)
                print(json.dumps({"point": "decode", "model": model, "size": size, "layers": TIPEZEN_LAYERS, "batch": b,
                                  "context": round(run["mean_context"]), "tok_s": round(run["tok_s"], 1),
                                  "ms_per_step": round(run["ms_per_step"], 4), "launches_per_step": run["launches"] // steps,
                                  **experts_of(engine, run["last_tokens"])}), flush=True)
            del engine
            torch.cuda.empty_cache()
            engine, cfg = make(size, 8, 8 * (P + 64), False, P)
            kinds = traced_kinds(engine, P, 8)
            line = {"point": "kernels", "model": model, "size": size, "prefill_tokens": P, "decode_batch": 8,
                    "prefill_ms_by_kind": kinds.get("prefill"), "decode_ms_by_kind": kinds.get("decode"), "peaks": peaks["source"]}
            if model == "kadodra":
                nl = TIPEZEN_LAYERS // 2                        # runs of either kind of layer
                gnorm_b = lambda T: nl * T * LH * LV * (4 + 4 + 2)
                finish_b = lambda T: nl * T * ((H * (D + R) + KR + R) * 4 + H * (D + R) * 2 + (KR + R) * 2 * (2 if T == P else 1))
                combine_b = lambda T: nl * T * W * (TOP * 4 + 4 + 4)
                spread_b = lambda T: nl * T * TOP * W * (2 + 2)
                norm_b = lambda T: (2 * nl * T + 1) * W * (4 + 2)
                fr = {}
                for step, T in (("prefill", P), ("decode", 8)):
                    k = kinds.get(step) or {}
                    for kind, nbytes in (("gated_norm", gnorm_b(T)), ("latent_finish", finish_b(T)), ("moe_combine", combine_b(T)),
                                         ("moe_spread", spread_b(T)), ("rmsnorm", norm_b(T))):
                        if kind in k:
                            fr[f"{step}_{kind}_hbm_frac"] = round(nbytes / (k[kind][1] / 1e3) / 1e9 / peaks["hbm_gbs"], 4)
                k = kinds.get("prefill") or {}
                if "retention_raw" in k:          # chunks of 64 tokens: A = Q K^T and A V, U = K^T V and Q S
                    flops = nl * LH * (P / 64.0) * 2.0 * 64 * (64 * LD + 64 * LV + 2 * LD * LV)
                    fr["prefill_retention_raw_fp32_tflops"] = round(flops / (k["retention_raw"][1] / 1e3) / 1e12, 2)
                if "attention_dense" in k:
                    span = min(WIN, P)
                    pairs = span * (span + 1) / 2.0 + (P - span) * span
                    fr["prefill_attention_dense_tflops"] = round(nl * H * pairs * 2.0 * (D + R + VD) / (k["attention_dense"][1] / 1e3) / 1e12, 2)
                if "gemm_tc_grouped" in k:
                    fr["prefill_experts_tcgen05_tflops"] = round(nl * P * TOP * 3 * 2.0 * W * F / (k["gemm_tc_grouped"][1] / 1e3) / 1e12, 2)
                    fr["prefill_experts_tcgen05_frac"] = round(fr["prefill_experts_tcgen05_tflops"] / peaks["bf16_tflops"], 4)
                if "gemm_tc" in k:                # lightning in and out, latent down and out, dense down; the up product is gemm_act
                    flops = nl * P * 2.0 * W * (2 * LH * LD + 3 * LH * LV + H * (D + R) + KR + R + H * VD + DF)
                    fr["prefill_dense_products_frac"] = round(flops / (k["gemm_tc"][1] / 1e3) / 1e12 / peaks["bf16_tflops"], 4)
                if "gemm_act" in k:
                    fr["prefill_gemm_act_frac"] = round(nl * P * 2.0 * W * DF / (k["gemm_act"][1] / 1e3) / 1e12 / peaks["bf16_tflops"], 4)
                kd = kinds.get("decode") or {}
                if "retention_raw" in kd:
                    fr["decode_retention_raw_hbm_frac"] = round(nl * 8 * LH * LD * LV * 4 * 2 / (kd["retention_raw"][1] / 1e3) / 1e9 / peaks["hbm_gbs"], 4)
                if "attention_tile" in kd:
                    fr["decode_attention_tile_hbm_frac"] = round(nl * 8 * min(WIN, P) * (KR + R) * 2 / (kd["attention_tile"][1] / 1e3) / 1e9 / peaks["hbm_gbs"], 4)
                if "gemm_grouped" in kd:          # the experts that 8 tokens of random ids touch, and the heads' projections
                    touched = experts_of(engine, [(7919 * i + 2) % TIPEZEN_VOCAB for i in range(8)])["experts_touched"]
                    w_b = nl * (touched * 3 * W * F * 2 + H * KR * (D + VD) * 2)
                    fr["decode_experts_touched"] = touched
                    fr["decode_gemm_grouped_hbm_frac"] = round(w_b / (kd["gemm_grouped"][1] / 1e3) / 1e9 / peaks["hbm_gbs"], 4)
                line["fractions"] = fr
            print(json.dumps(line), flush=True)
            del engine
            torch.cuda.empty_cache()
    clocks.stop()
    print(json.dumps({"point": "clocks", "clocks": clocks.summary()}), flush=True)
    return 0


# The Gumodra design beside Kadodra (the closest of the other models: one norm for two sublayers side by side, a windowed
# attention with a learned sink and linear attention over matrix states in turn, dense and routed feed-forwards) at the same
# width: (width, attention heads, kv heads, dim, window, kept first tokens, mlstm heads, key size, value size, experts, chosen,
# groups, kept groups, expert ff, shared ff, dense ff).  Eight layers, mlstm with a dense feed-forward and attention with experts
# in turn; the dense feed-forward is gated, so its ff is two thirds of the twin's for the same arithmetic.  What the twin has no
# like of: the gates of the residual (two width x width products a layer) and the shared expert.
GUMODRA_SIZES = {"2k": (2048, 16, 4, 128, 1024, 64, 16, 128, 128, 16, 2, 4, 2, 3072, 3072, 6144),
                 "4k": (4096, 32, 8, 128, 1024, 64, 32, 128, 128, 16, 2, 4, 2, 6144, 6144, 12288)}


def gumodra_engine(size: str, max_live: int, cache_tokens: int, graphs: bool, step_tokens: int):
    import torch
    import tffinfer_b200 as tff
    from tffinfer_b200.config.gumodra_config import GumodraConfig, GumodraLayer, GumodraMlp, GumodraAttention, GumodraMlstm
    from tffinfer_b200.config.tipezen_config import RotaryConfig
    from tffinfer_b200.weights import random_tensors_on_device
    W, H, G, D, WIN, KEEP, MH, MD, MV, E, TOP, NG, KG, F, SF, DF = GUMODRA_SIZES[size]
    memory = GumodraLayer("mlstm", mlp=GumodraMlp("dense", DF), mlstm=GumodraMlstm(MH, MD, MV, 15.0))
    attention = GumodraLayer("attention", mlp=GumodraMlp("moe", F, E, TOP, (NG, KG), SF), attention=GumodraAttention(
        H, G, D, D ** -0.5, RotaryConfig(5e5, D // 2), WIN, KEEP))
    cfg = GumodraConfig("Gumodra", vocab_size=TIPEZEN_VOCAB, hidden_size=W, norm_eps=1e-6, embed_scale=W ** 0.5,
                        layers=(memory, attention) * (TIPEZEN_LAYERS // 2))
    tensors = random_tensors_on_device(cfg, 0, "cuda", "bfloat16")
    ecfg = tff.EngineConfig(dtype="bfloat16", page_size=PAGE_SIZE, max_cache_tokens=cache_tokens, max_live_requests=max_live,
                            max_tokens_per_step=step_tokens, max_model_len=8192, use_cuda_graphs=graphs)
    runner = tff.ModelRunner(config=cfg, tensors=tensors, engine_config=ecfg)
    del tensors
    torch.cuda.empty_cache()
    return tff.Engine(runner=runner), cfg


def run_gumodra(steps: int, warmup: int, sizes=None) -> int:
    """Prefill and decode throughput of the Gumodra design beside Kadodra at the same layer sizes, one JSON line a point, and
    for each model the device time of a step by kind of kernel call; for Gumodra also what its own kernels reach: the mLSTM
    recurrence in TFLOP/s of its chunk form (prompt step) and as a fraction of the measured copy rate for the states it reads
    and writes (decode step), the windowed attention, the kernels of the residual's gates, of the heads, of the norm behind the
    recurrence and of the experts' sum as fractions of the copy rate, the products of the measured bfloat16 rate."""
    import torch
    peaks = load_peaks()
    steps = min(steps, 32)
    P = PROMPT_LEN
    clocks = ClockSampler()
    clocks.start()
    for size in (sizes or GUMODRA_SIZES):
        W, H, G, D, WIN, KEEP, MH, MD, MV, E, TOP, NG, KG, F, SF, DF = GUMODRA_SIZES[size]
        for model, make in (("gumodra", gumodra_engine), ("kadodra", kadodra_engine)):
            need = 64 * (P + warmup + steps + 64 + 72)
            engine, cfg = make(size, 64, need, True, P)
            pms = prefill_run(engine, iters=3, warmup=2, seed=1, prompt_len=P)
            print(json.dumps({"point": "prefill", "model": model, "size": size, "layers": TIPEZEN_LAYERS, "tokens": P,
                              "ms": round(pms, 3), "tok_s": round(P / (pms / 1e3), 1)}), flush=True)
            for b in (8, 64):
                run = decode_run(engine, b, steps, warmup, seed=b, prompt_len=P)
                print(json.dumps({"point": "decode", "model": model, "size": size, "layers": TIPEZEN_LAYERS, "batch": b,
                                  "context": round(run["mean_context"]), "tok_s": round(run["tok_s"], 1),
                                  "ms_per_step": round(run["ms_per_step"], 4), "launches_per_step": run["launches"] // steps,
                                  **experts_of(engine, run["last_tokens"])}), flush=True)
            del engine
            torch.cuda.empty_cache()
            engine, cfg = make(size, 8, 8 * (P + 64), False, P)
            kinds = traced_kinds(engine, P, 8)
            line = {"point": "kernels", "model": model, "size": size, "prefill_tokens": P, "decode_batch": 8,
                    "prefill_ms_by_kind": kinds.get("prefill"), "decode_ms_by_kind": kinds.get("decode"), "peaks": peaks["source"]}
            if model == "gumodra":
                nl = TIPEZEN_LAYERS // 2                        # layers of either kind
                fr = {}
                for step, T in (("prefill", P), ("decode", 8)):
                    k = kinds.get(step) or {}
                    z = 2 if T == P else 4                      # bytes of a gate: bfloat16 in prompts, accumulators in decode steps
                    for kind, nbytes in (("gated_join", (2 * nl - 1) * T * W * (4 + 4 + 4 + 4 + 2 * z + 2)),
                                         ("gated_norm", nl * T * MH * MV * (4 + 4 + 2)),
                                         ("qk_finish", nl * T * D * ((H + G) * 4 + (H + 2 * G) * 2)),
                                         ("moe_combine", nl * T * W * (TOP * 4 + 4 + 4))):
                        if kind in k:
                            fr[f"{step}_{kind}_hbm_frac"] = round(nbytes / (k[kind][1] / 1e3) / 1e9 / peaks["hbm_gbs"], 4)
                k, kd = kinds.get("prefill") or {}, kinds.get("decode") or {}
                if "mlstm_recurrence" in k:       # chunks of 64 tokens: A = Q K^T and A V, U = K^T V and Q S
                    flops = nl * MH * (P / 64.0) * 2.0 * 64 * (64 * MD + 64 * MV + 2 * MD * MV)
                    fr["prefill_mlstm_recurrence_tflops"] = round(flops / (k["mlstm_recurrence"][1] / 1e3) / 1e12, 2)
                if "attention_bf16" in k:
                    span = min(WIN, P)
                    pairs = span * (span + 1) / 2.0 + (P - span) * (span + KEEP)
                    fr["prefill_attention_bf16_tflops"] = round(nl * H * pairs * 4.0 * D / (k["attention_bf16"][1] / 1e3) / 1e12, 2)
                if "gemm_tc_grouped" in k:
                    fr["prefill_experts_tcgen05_frac"] = round(nl * P * TOP * 6.0 * W * F / (k["gemm_tc_grouped"][1] / 1e3) / 1e12 / peaks["bf16_tflops"], 4)
                if "gemm_tc" in k:                # mlstm in and out, attention in and out, gates, both down products
                    flops = P * 2.0 * W * (nl * (2 * MH * MD + 3 * MH * MV + 2 * MH + (2 * H + G) * D + SF + DF) + 2 * nl * 2 * W)
                    fr["prefill_dense_products_frac"] = round(flops / (k["gemm_tc"][1] / 1e3) / 1e12 / peaks["bf16_tflops"], 4)
                if "gemm_gated_act" in k:
                    fr["prefill_gemm_gated_act_frac"] = round(nl * P * 4.0 * W * (DF + SF) / (k["gemm_gated_act"][1] / 1e3) / 1e12 / peaks["bf16_tflops"], 4)
                if "mlstm_recurrence" in kd:
                    fr["decode_mlstm_recurrence_hbm_frac"] = round(nl * 8 * MH * MD * (MV + 1) * 4 * 2 / (kd["mlstm_recurrence"][1] / 1e3) / 1e9 / peaks["hbm_gbs"], 4)
                if "attention_bf16" in kd:
                    fr["decode_attention_bf16_hbm_frac"] = round(nl * 8 * min(WIN + KEEP, P) * 2 * G * D * 2 / (kd["attention_bf16"][1] / 1e3) / 1e9 / peaks["hbm_gbs"], 4)
                line["fractions"] = fr
            print(json.dumps(line), flush=True)
            del engine
            torch.cuda.empty_cache()
    clocks.stop()
    print(json.dumps({"point": "clocks", "clocks": clocks.summary()}), flush=True)
    return 0


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--workload", default="headline", choices=["headline", "sweep", "attn_decode", "shapes", "tipezen", "dominex", "sadupel", "nugosun", "kadodra", "gumodra"] + sorted(WORKLOADS),
                    help="headline: the decode/prefill benchmark; sweep: the same shape at further batch sizes and "
                         "context lengths; attn_decode: the decode attention alone; shapes: the layer sizes of the other "
                         "models of the family; tipezen: the Tipezen design beside Qwen3 at equal layer sizes; dominex: the Dominex design beside Tipezen at equal layer sizes; sadupel: the Sadupel design beside Dominex at equal layer sizes; nugosun: the Nugosun design beside Dominex at equal layer sizes; kadodra: the Kadodra design beside Nugosun at equal layer sizes; gumodra: the Gumodra design beside Kadodra at equal layer sizes; else a whole workload through "
                         "the scheduler")
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=4)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--size", default="", help="with --workload dominex, sadupel, nugosun, kadodra or gumodra: one of its layer sizes (2k, 4k) instead of all")
    ap.add_argument("--layers", type=int, default=SHAPE["num_layers"],
                    help="fewer layers than the shape has (both numbers are reported)")
    ap.add_argument("--skip-points", action="store_true", help="only the headline batch (no batch 1 / 64, no prefill)")
    ap.add_argument("--no-graphs", action="store_true", help="launch decode steps kernel by kernel (for profilers)")
    args = ap.parse_args()

    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable":
                          "NKKdev/TFFinfer is a CMake C++/CUDA project without Python packaging whose dependencies "
                          "(glog, Taskflow, libdivide) are fetched from the network; it loads GGUF Q8_0 files only and "
                          "has no sm_100 build: it cannot be installed offline here"}))
        return 0
    if args.gpus != 1:
        print(f"bench.py: this engine runs on one GPU; --gpus {args.gpus} is not supported")
        return 2
    warmup = max(3, args.warmup)
    if args.workload == "sweep":
        return run_sweep(args.layers, args.steps, warmup)
    if args.workload == "attn_decode":
        return run_attn_decode()
    if args.workload == "shapes":
        return run_shapes(args.steps, warmup)
    if args.workload == "tipezen":
        return run_tipezen(args.steps, warmup)
    if args.workload == "dominex":
        return run_dominex(args.steps, warmup, [args.size] if args.size else None)
    if args.workload == "sadupel":
        return run_sadupel(args.steps, warmup, [args.size] if args.size else None)
    if args.workload == "nugosun":
        return run_nugosun(args.steps, warmup, [args.size] if args.size else None)
    if args.workload == "kadodra":
        return run_kadodra(args.steps, warmup, [args.size] if args.size else None)
    if args.workload == "gumodra":
        return run_gumodra(args.steps, warmup, [args.size] if args.size else None)
    if args.workload != "headline":
        return run_workload(args.workload, 0 if args.layers == SHAPE["num_layers"] else args.layers)

    import torch
    if not torch.cuda.is_available():
        print("bench.py: no CUDA device", file=sys.stderr)
        return 1
    peaks = load_peaks()
    max_batch = args.batch if args.skip_points else max(args.batch, 64)
    tokens_needed = max_batch * (PROMPT_LEN + warmup + args.steps + max_batch + 64)
    engine, cfg = make_engine(args.layers, max_batch, tokens_needed, graphs=not args.no_graphs)
    mb = model_bytes(cfg)

    clocks = ClockSampler()
    main_run = decode_run(engine, args.batch, args.steps, warmup, seed=1, sampler=clocks)
    points = {}
    points_roofline = {}
    prefill = None

    def hbm_fraction(run, batch):
        """bytes the step has to read (every weight once, the cache of the live requests) / its time / the peak"""
        b = mb["weights_read_per_step"] + batch * run["mean_context"] * mb["kv_bytes_per_token"]
        return b / (run["ms_per_step"] / 1e3) / 1e9 / peaks["hbm_gbs"]

    if not args.skip_points:
        small_steps = min(args.steps, 32)
        for name, b, seed in (("decode_b1", 1, 2), ("decode_b64", 64, 3)):
            run = decode_run(engine, b, small_steps, warmup, seed=seed)
            points[name] = round(run["tok_s"], 1)
            points_roofline[name] = {"ms_per_step": round(run["ms_per_step"], 4), "hbm_frac": round(hbm_fraction(run, b), 4),
                                     "p50_ms": round(run["p50_ms"], 4), "p99_ms": round(run["p99_ms"], 4)}
        pms = prefill_run(engine, iters=5, warmup=3, seed=4)
        T = PROMPT_LEN
        flops = prefill_flops(cfg, mb, T)
        prefill = {"value": round(T / (pms / 1e3), 1), "tokens": T, "ms": round(pms, 3),
                   "frac": round(flops / (pms / 1e3) / (peaks["bf16_tflops"] * 1e12), 4),
                   "tflops": round(flops / (pms / 1e3) / 1e12, 1)}

    step_s = main_run["ms_per_step"] / 1e3
    bytes_step = mb["weights_read_per_step"] + args.batch * main_run["mean_context"] * mb["kv_bytes_per_token"]
    achieved = bytes_step / step_s / 1e9
    out = {
        "metric": "decode tok/s (Qwen3-8B shape, bf16, batch 8, 2048-token prompts)",
        "value": round(main_run["tok_s"], 1), "unit": "tok/s", "n_gpus": 1, "steps": args.steps, "warmup": warmup,
        "ms_per_step": round(main_run["ms_per_step"], 4), "higher_is_better": True, "scaling": "weak",
        "vs_baseline": None, "dtype": "bf16", "data": "synthetic (seeded uniform token ids, random N(0,0.02) weights)",
        "impl": "ours",
        "config": {"model": "Qwen3-8B shape", "layers": cfg.num_layers, "layers_of_shape": SHAPE["num_layers"],
                   "hidden": cfg.hidden_size, "heads": cfg.num_heads, "kv_heads": cfg.num_kv_heads,
                   "head_dim": cfg.head_dim, "intermediate": cfg.intermediate_size, "vocab": cfg.vocab_size,
                   "global_batch": args.batch, "seq_len": CONTEXT, "prompt_len": PROMPT_LEN, "page_size": PAGE_SIZE,
                   "parallelism": "1 GPU", "l2": "inputs larger than L2 (15 GB of weights read per step)",
                   "cuda_graphs": not args.no_graphs},
        "e2e": {"value": round(main_run["e2e_tok_s"], 1), "unit": "tok/s",
                "h2d_bytes_per_step": main_run["h2d_bytes"], "d2h_bytes_per_step": main_run["d2h_bytes"]},
        "gpu_launches": main_run["launches"],
        "latency_ms": {"p50": round(main_run["p50_ms"], 4), "p99": round(main_run["p99_ms"], 4),
                       "max": round(main_run["max_ms"], 4)},
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": peaks["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / peaks["hbm_gbs"], 4), "peaks": peaks["source"]},
        "clocks": clocks.summary(),
    }
    if prefill is not None:
        out["prefill"] = prefill
        out["points"] = points
        out["points_roofline"] = points_roofline
    print(json.dumps(out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
