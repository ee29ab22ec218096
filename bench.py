"""Benchmark of the pih_b200 engine: decode tokens per second of Qwen3-0.6B on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--batch 8] [--impl ours|reference]

A "step" is one decode step of the batch.  The default run has the layer
sizes of the Qwen3-0.6B configuration (28 layers, hidden 1024, 16/8 heads of
128, intermediate 3072, vocabulary 151 936, tied embeddings) with random
weights (N(0, 0.02), seed 2), a batch of 8 requests each holding 2 048
context tokens, page size 64.  It prints ONE JSON line:

* ``value``      decoded tokens per second, timed on the device with CUDA events around K
                 steps of the step function plus device sampling (no host transfer inside);
* ``e2e``        the same through the Python entry point (``Engine.step``): every step packs its
                 batch on the host, copies it from pinned memory, and reads the sampled tokens back;
* ``prefill``    one 2 048-token prompt in one step: tokens/s, ms, and the fraction of the bf16 peak, for the step
                 replayed from its CUDA graph (a shape seen before), and ``first_sight_ms`` for the same step at
                 the first sight of its shape, launched kernel by kernel;
* ``roofline``   bytes a decode step has to read (every weight once, the cache of the live
                 requests) / its time, against the measured HBM copy bandwidth;
* ``points``     decode tokens/s at batch 1 and 64.

Peaks come from MEASURED_PEAKS.json beside this file if it exists, else the
fallback 6.65 TB/s and 1.59 PFLOP/s.  Inputs (1.2 GB of weights plus the
cache) are larger than the 126 MB L2, so no flush is needed between steps.
"""
from __future__ import annotations

import argparse
import gc
import json
import os
import subprocess
import sys
import tempfile
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

QWEN3_0_6B = {
    "architectures": ["Qwen3ForCausalLM"], "model_type": "qwen3", "torch_dtype": "bfloat16",
    "hidden_act": "silu", "use_cache": True, "tie_word_embeddings": True,
    "hidden_size": 1024, "intermediate_size": 3072, "num_hidden_layers": 28,
    "num_attention_heads": 16, "num_key_value_heads": 8, "head_dim": 128, "vocab_size": 151936,
    "max_position_embeddings": 40960, "rope_theta": 1000000.0, "rms_norm_eps": 1e-6,
    "bos_token_id": 151643, "eos_token_id": 151645, "attention_bias": False, "use_sliding_window": False,
}
CONTEXT = 2048
PREFILL_TOKENS = 2048
PAGE = 64
METRIC = "decode tok/s at batch 8 (Qwen3-0.6B, 2048-token contexts)"


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    hbm, flops, src = 6650.0, 1590.0, "fallback"
    def number(v, default):
        if isinstance(v, dict):                      # {"value": ...} or the like
            v = next((v[k] for k in ("value", "median", "mean") if k in v), None)
        try:
            v = float(v)
        except (TypeError, ValueError):
            return default
        return v if v > 0 else default

    try:
        with open(path) as f:
            p = json.load(f)
        if isinstance(p, dict):
            measured_hbm, measured_flops = number(p.get("hbm_gbs"), None), number(p.get("bf16_tflops"), None)
            if measured_hbm is not None and measured_flops is not None:
                hbm, flops, src = measured_hbm, measured_flops, "measured"
    except (OSError, ValueError):
        pass
    return hbm, flops, src


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while the timed region runs."""
    QUERY = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, index: int = 0):
        self.samples = []
        self._stop = threading.Event()
        self._proc = None
        self._thread = None
        self.index = index

    def __enter__(self):
        try:
            self._proc = subprocess.Popen(
                ["nvidia-smi", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits", "-lms", "100",
                 "-i", str(self.index)], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            self._thread = threading.Thread(target=self._read, daemon=True)
            self._thread.start()
        except OSError:
            self._proc = None
        return self

    def _read(self):
        for line in self._proc.stdout:
            parts = [p.strip() for p in line.split(",")]
            if len(parts) == 6 and parts[0].isdigit():
                self.samples.append(parts)
            if self._stop.is_set():
                break

    def __exit__(self, *exc):
        self._stop.set()
        if self._proc is not None:
            self._proc.terminate()
            try:
                self._proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self._proc.kill()

    def summary(self):
        if not self.samples:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["no samples"]}
        mhz = sorted(int(s[0]) for s in self.samples)
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = [n for i, n in enumerate(names) if any(s[2 + i].lower().startswith("active") for s in self.samples)]
        return {"sm_mhz": mhz[len(mhz) // 2], "sm_max_mhz": int(self.samples[0][1]), "reasons": reasons,
                "samples": len(mhz)}


def build_model(layers: int):
    import torch
    from pih_b200.config import config_from_dict
    from pih_b200.kernels import get_ops
    from pih_b200.models import CausalLM, expected_tensors
    from pih_b200.parts import Runtime
    from pih_b200.weights import random_tensors

    raw = dict(QWEN3_0_6B, num_hidden_layers=layers)
    config = config_from_dict(raw)
    spec = config.model_spec()
    dev = torch.device("cuda:0")
    rt = Runtime(dev, torch.bfloat16, get_ops(dev))
    weights = random_tensors(expected_tensors(spec), seed=2, sigma=0.02, dtype=torch.bfloat16)
    return config, CausalLM(spec, weights, rt)


def weight_bytes(model) -> int:
    """Bytes of every weight a decode step reads once (the embedding table counts as the tied head)."""
    seen, total = set(), 0
    tensors = [model.head]
    for b in model.blocks:
        tensors += [b.mixer.w_qkv, b.mixer.w_o, b.ffn.w_gate_up, b.ffn.w_down, b.norm_in.weight,
                    b.norm_post.weight, b.mixer.q_norm, b.mixer.k_norm]
    tensors.append(model.final_norm.weight)
    for t in tensors:
        if t is not None and t.data_ptr() not in seen:
            seen.add(t.data_ptr())
            total += t.numel() * t.element_size()
    return total


def decode_run(model, batch: int, steps: int, warmup: int, context: int = CONTEXT, repeats: int = 5):
    """Device-timed decode: ``batch`` requests with ``context`` tokens in the cache
    (synthetic keys and values), one token each per step, greedy sampling on the device.  The timed loop of
    ``steps`` steps runs ``repeats`` times back to back; the median loop is reported."""
    import torch
    from pih_b200.cache import CacheManager
    from pih_b200.engine import ModelRunner, StepEntry

    spec = model.spec
    rt = model.rt
    total = steps * repeats + warmup
    cache = CacheManager(model.cache_needs(), [e.reads_cache_of for e in spec.schedule], page_size=PAGE,
                         num_pages=batch * (-(-(context + total + 1) // PAGE)), max_requests=batch,
                         device=rt.device, dtype=rt.dtype)
    for grp in cache.groups:
        grp.kv.normal_(0.0, 1.0)
    for r in range(batch):
        cache.add_request(r)
        cache.append(r, context)
        cache.commit(r)
    runner = ModelRunner(model, cache, cuda_graphs=True)
    g = torch.Generator().manual_seed(5)
    tokens = torch.randint(0, spec.vocab, (batch,), generator=g).tolist()

    def one_step(tokens):
        logits = runner.step([StepEntry(r, [tokens[r]], [0]) for r in range(batch)])
        return rt.ops.argmax(logits)

    for _ in range(warmup):
        tokens = one_step(tokens).tolist()
    loops = []
    for _ in range(repeats):
        torch.cuda.synchronize()
        launches0 = rt.ops.launches
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        # timed: the next token ids are kept as given (host list) so that no D2H sits in the region
        start.record()
        for _ in range(steps):
            out = one_step(tokens)
        stop.record()
        torch.cuda.synchronize()
        loops.append((start.elapsed_time(stop) / steps, rt.ops.launches - launches0, cache.requests[0].num_tokens))
    rt.ops.check_errors()
    ms, launches, length_after = sorted(loops)[len(loops) // 2]
    kv_bytes = batch * (length_after - steps // 2) * cache.bytes_per_token()
    del out
    for r in range(batch):
        cache.release(r)
    return {"ms": ms, "tok_s": batch / ms * 1e3, "launches": launches, "bytes": weight_bytes(model) + kv_bytes,
            "loops_ms": [round(l[0], 4) for l in loops]}


def prefill_run(model, tokens_n: int, reps: int = 6):
    import torch
    from pih_b200.cache import CacheManager
    from pih_b200.engine import ModelRunner, StepEntry

    spec, rt = model.spec, model.rt
    cache = CacheManager(model.cache_needs(), [e.reads_cache_of for e in spec.schedule], page_size=PAGE,
                         num_pages=-(-tokens_n // PAGE) + 1, max_requests=1, device=rt.device, dtype=rt.dtype)
    runner = ModelRunner(model, cache, cuda_graphs=True)    # a repeated portion shape is replayed from a graph
    g = torch.Generator().manual_seed(6)
    toks = torch.randint(0, spec.vocab, (tokens_n,), generator=g).tolist()
    # prompts of other lengths first: what the kernels and the library set up or load at their first calls with
    # rows of about this number is not part of "the first sight of a shape" in a process that has served before
    for cut in (48, 112, 16, 80):
        runner.step([StepEntry("w", toks[:tokens_n - cut], [tokens_n - cut - 1])])
        torch.cuda.synchronize()
        runner.finish("w")
    times = []
    first_sight = None
    for i in range(reps + 2):
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        start.record()
        runner.step([StepEntry("p", toks, [tokens_n - 1])])
        stop.record()
        torch.cuda.synchronize()
        runner.finish("p")
        if i == 0:                                           # a shape not seen before: run as it is, launch by launch
            first_sight = start.elapsed_time(stop)
        if i >= 2:                                           # (the second run captures)
            times.append(start.elapsed_time(stop))
    rt.ops.check_errors()
    ms = sorted(times)[len(times) // 2]
    # flops: 2 * tokens * linear parameters + causal attention (QK^T and PV) + one row of the head
    lin = sum(t.numel() for b in model.blocks for t in (b.mixer.w_qkv, b.mixer.w_o, b.ffn.w_gate_up, b.ffn.w_down))
    a = model.blocks[0].mixer.spec
    attn = len(model.blocks) * 4 * a.heads * a.head_dim * tokens_n * (tokens_n + 1) // 2
    flops = 2 * tokens_n * lin + attn + 2 * model.head.numel()
    return {"ms": ms, "tok_s": tokens_n / ms * 1e3, "flops": flops, "first_sight_ms": first_sight}


def e2e_run(config, model_dir_weights, batch: int, steps: int, warmup: int):
    """Through the Python entry point: submit prompts, let the engine prefill, then time decode steps
    wall-clock; each step packs and copies its batch from pinned host memory and reads tokens back."""
    import torch
    from pih_b200.engine import Engine
    from pih_b200.sampling import SamplingParams

    engine = Engine(model_dir_weights, "bfloat16", page_size=PAGE, maximum_batch_sequences=batch,
                    maximum_batch_tokens=4096, maximum_context_tokens=2 * CONTEXT,    # the pool: sized by the engine
                    capture_decode_after=0)        # the batch never changes: its graph is captured at once
    g = torch.Generator().manual_seed(7)
    # long enough that no request finishes inside the timed region (prompts finish prefill on different steps)
    params = SamplingParams(max_tokens=steps + warmup + batch + 16, ignore_eos=True)
    reqs = []
    for _ in range(batch):
        rid = engine.submit(torch.randint(0, config.vocab_size, (CONTEXT,), generator=g).tolist(), params)
        reqs.append(engine._live[rid])
    while any(r.num_computed < len(r.prompt) for r in reqs):
        engine.step()
    for _ in range(warmup - 1):
        engine.step()
    torch.cuda.synchronize()
    # what the process has allocated so far (weights' tensor lists, the earlier runs' graphs) is set aside, as a
    # serving process does after start-up: a full collection over it inside the timed steps is a pause of
    # milliseconds that belongs to this script's earlier runs, not to a step
    gc.collect()
    gc.freeze()
    before = sum(len(r.outputs) for r in reqs)
    t0 = time.perf_counter()
    for _ in range(steps):
        engine.step()
    torch.cuda.synchronize()
    dt = time.perf_counter() - t0
    gc.unfreeze()
    produced = sum(len(r.outputs) for r in reqs) - before
    assert produced == batch * steps, (produced, batch, steps)
    h2d = engine.runner.builder.last_bytes
    return {"value": produced / dt, "unit": "tok/s", "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": 4 * batch,
            "ms_per_step": dt / steps * 1e3}


# -- the Rigotar design beside the dense decoder at equal width ---------------------------------------------------
def _rigotar_config(width: int, layers: int, kinds=("rglru", "latent_attention", "delta", "latent_attention"), moe=True,
                    vocab: int = 32768):
    """Layer sizes that resemble a real model's at this width: 128-wide heads, a latent of a quarter of the width,
    sixteen experts of which two are used, with as many active feed-forward weights as the dense model's."""
    heads = width // 128
    mixers = {"delta": {"heads": heads, "kv_heads": max(1, heads // 2), "dim": 128, "vdim": 128, "conv": 4},
              "rglru": {"width": width, "blocks": heads, "conv": 4},
              "latent_attention": {"heads": heads, "dim": 128, "vdim": 128, "kv_rank": width // 4, "scale": 128 ** -0.5}}
    mlp = {"kind": "moe", "router": {"experts": 16, "top": 2}, "expert": {"ff": 3 * width // 2}} if moe else None
    return {"architecture": "Rigotar", "vocab": vocab, "width": width, "norm": {"eps": 1e-6},
            "layers": [{"type": kinds[i % len(kinds)], "mixer": mixers[kinds[i % len(kinds)]], "mlp": mlp}
                       for i in range(layers)]}


def _tuganex_config(width: int, layers: int, kinds=("attention", "retention"), mlps=("dense", "moe"), vocab: int = 32768,
                    share_from: int = -1):
    """Layer sizes that resemble a real model's at this width: heads of two 64-wide maps (128-wide retention keys) and
    128-wide values, half as many key/value heads, a dense feed-forward of three times the width, and sixteen experts
    with two identity experts in three groups of which two are kept, two chosen, and a shared expert.  ``share_from``:
    from this layer on, attention layers read the keys and values of the first attention layer."""
    heads = width // 128
    rot = {"dims": 64, "base": 1e6}
    mixers = {"attention": {"heads": heads, "kv_heads": max(1, heads // 2), "dim": 64, "vdim": 128, "rot": rot,
                            "scale": 0.125, "diff": 0.5},
              "retention": {"heads": heads, "dim": 128, "vdim": 128, "rot": rot,
                            "decay": [1.0 - 2.0 ** (-5 - 5 * h / max(1, heads - 1)) for h in range(heads)]}}
    ffs = {"dense": {"kind": "dense", "ff": 3 * width}, None: None,
           "moe": {"kind": "moe", "router": {"experts": 16, "identity": 2, "top": 2, "groups": {"count": 3, "keep": 2}},
                   "expert": {"ff": 3 * width // 2}, "shared": {"ff": width // 2}}}
    out, first_attention = [], None
    for i in range(layers):
        kind = kinds[i % len(kinds)]
        mixer = dict(mixers[kind])
        if kind == "attention":
            if first_attention is None:
                first_attention = i
            elif 0 <= share_from <= i:
                mixer["kv_from"] = first_attention
        out.append({"type": kind, "mixer": mixer, "mlp": ffs[mlps[(i // len(kinds)) % len(mlps)] if mlps else None]})
    return {"architecture": "Tuganex", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "layers": out}


def _pegopel_config(width: int, layers: int, kinds=("attention", "attention_2"), window: int = 1024, keep_first: int = 64,
                    mlp: bool = True, streams: int = 2, loop=None, vocab: int = 32768):
    """Layer sizes that resemble a real model's at this width: 128-wide heads, half as many key/value heads (the dense
    decoder's), windows of ``window`` keys (beyond the context: every key is seen, as in the dense decoder), four-tap
    convolutions and a bias table of 32 rows on the one mixer; a stretched rotation over half of each head, capped
    scores, ``keep_first`` kept tokens and the head gates on the other; a feed-forward of three times the width; two
    residual streams."""
    heads = width // 128 * 2
    common = {"heads": heads, "kv_heads": max(1, heads // 2), "dim": 128, "vdim": 128, "scale": 128 ** -0.5}
    mixers = {"attention": dict(common, conv=4, bias_max=float(2 * window), bias_rows=32, mask={"size": window}),
              "attention_2": dict(common, softcap=30.0, mask={"size": window, "keep_first": keep_first},
                                  rot={"dims": 64, "base": 1e6, "scaling": {"factor": 4.0, "original": 2048, "fast": 32.0,
                                                                            "slow": 1.0}})}
    out = {"architecture": "Pegopel", "vocab": vocab, "width": width, "max_positions": 8192, "norm": {"eps": 1e-6},
           "layers": [{"type": kinds[i % len(kinds)], "mixer": mixers[kinds[i % len(kinds)]],
                       "mlp": {"kind": "dense", "ff": 3 * width} if mlp else None} for i in range(layers)]}
    if streams:
        out["streams"] = streams
    if loop is not None:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


def _sagelorn_config(width: int, layers: int, kinds=("attention", "latent_attention", "attention", "retention"),
                     mlps=("dense", "moe"), window: int = 1024, share: bool = True, vocab: int = 32768):
    """Layer sizes that resemble a real model's at this width: 128-wide heads with half as many key/value heads, a
    rotation over half of each head with stretched slow pairs and windows of ``window`` keys on the attention (every
    second attention layer reads the keys and values of the one before it, with ``share``); latent attention with as
    many heads as Rigotar's (one a 128 of the width), a latent and 64 rotated numbers that are a quarter of the width
    together, queries through a latent of half the width; 128-wide retention heads; a dense feed-forward of three times the width, and sixteen two-matrix experts of twice the width of which two
    are chosen, with a shared expert of half the width: as many active feed-forward weights as the dense one."""
    heads = width // 128 * 2
    rot = {"dims": 64, "base": 1e6, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 2048}}
    mixers = {"attention": {"heads": heads, "kv_heads": max(1, heads // 2), "dim": 128, "vdim": 128, "rot": rot,
                            "scale": 128 ** -0.5, "mask": {"size": window}},
              "latent_attention": {"heads": heads // 2, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": width // 4 - 64,
                                   "q_rank": width // 2, "rot": {"dims": 64, "base": 1e4}, "scale": 192 ** -0.5,
                                   "mask": {"size": window}},
              "retention": {"heads": heads // 2, "dim": 128, "vdim": 128,
                            "decay": [1.0 - 2.0 ** (-5 - 5 * h / max(1, heads // 2 - 1)) for h in range(heads // 2)]}}
    ffs = {"dense": {"kind": "dense", "ff": 3 * width}, None: None,
           "moe": {"kind": "moe", "router": {"experts": 16, "top": 2}, "expert": {"ff": 2 * width},
                   "shared": {"ff": width // 2}}}
    out, last_owner = [], None
    for i in range(layers):
        kind = kinds[i % len(kinds)]
        mixer = dict(mixers[kind])
        if kind == "attention":
            if share and last_owner is not None:
                mixer["kv_from"], last_owner = last_owner, None
            else:
                last_owner = i
        out.append({"type": kind, "mixer": mixer, "mlp": ffs[mlps[i % len(mlps)] if mlps else None]})
    return {"architecture": "Sagelorn", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "logit_scale": 0.5,
            "embedding": {"bigram": {"buckets": 65521, "mul_prev": 31, "mul_cur": 17}}, "layers": out}


def _kedavik_config(width: int, layers: int, kinds=("mamba1", "parallel"), mlp: bool = True, chunk: int = 1024, loop=None,
                    vocab: int = 32768):
    """Layer sizes that resemble a real model's at this width: a scan over twice the width with 16 states a channel and
    step sizes through a sixteenth of the width; beside each other half as many 128-wide attention heads as the dense
    decoder's (half as many key/value heads, whole heads rotated, chunks of ``chunk`` places) and as many 128 x 128 delta
    heads as Rigotar's, decays and gate through 128 numbers; a two-matrix feed-forward of four times the width behind the
    pair."""
    heads = width // 128
    mixers = {"mamba1": {"inner": 2 * width, "state": 16, "dt_rank": width // 16, "conv": 4},
              "parallel": {"left": {"heads": heads, "kv_heads": max(1, heads // 2), "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                                    "rot": {"dims": 128, "base": 1e6}, "mask": {"size": chunk}},
                           "right": {"heads": heads, "kv_heads": max(1, heads // 2), "dim": 128, "vdim": 128, "conv": 4,
                                     "decay_rank": 128, "gate_rank": 128}, "left_scale": 0.8, "right_scale": 0.6}}
    out = {"architecture": "Kedavik", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": 0.5},
           "residual_mult": 0.4,
           "layers": [{"type": kinds[i % len(kinds)], "mixer": mixers[kinds[i % len(kinds)]],
                       "mlp": {"kind": "dense", "ff": 4 * width} if mlp and kinds[i % len(kinds)] == "parallel" else None}
                      for i in range(layers)]}
    if loop is not None:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


def _bipulorn_config(width: int, layers: int, kinds=("gla", "parallel", "mlstm", "parallel"), moe: bool = True,
                     window: int = 1024, vocab: int = 32768):
    """Layer sizes that resemble a real model's at this width: a 128 x 128 matrix state a head and as many heads as
    Tuganex's retention for the two plain recurrences (decays through 16 numbers); beside each other as many 128-wide
    attention heads as Kedavik's (half as many key/value heads, half of each head rotated, windows of ``window`` keys) and a
    state-space dual layer of twice the width (64-wide heads, 128 states, one group); Tuganex's experts (sixteen and two
    identity experts, two chosen, a shared one)."""
    heads = width // 128
    mixers = {"gla": {"heads": heads, "dim": 128, "vdim": 128, "tau": 16.0, "decay_rank": 16},
              "mlstm": {"heads": heads, "dim": 128, "vdim": 128, "gate_cap": 15.0},
              "parallel": {"left": {"heads": heads, "kv_heads": max(1, heads // 2), "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                                    "rot": {"dims": 64, "base": 1e6, "scaling": {"factor": 4.0}}, "mask": {"size": window}},
                           "right": {"heads": 2 * width // 64, "vdim": 64, "state": 128, "groups": 1, "norm_groups": 1, "conv": 4}}}
    mlp = {"kind": "moe", "router": {"experts": 16, "identity": 2, "top": 2, "scale": 2.0}, "expert": {"ff": 3 * width // 2},
           "shared": {"ff": width // 2}} if moe else None
    return {"architecture": "Bipulorn", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "logit_softcap": 30.0,
            "layers": [{"type": kinds[i % len(kinds)], "mixer": mixers[kinds[i % len(kinds)]], "mlp": mlp} for i in range(layers)]}


def _dense_config(width: int, layers: int, vocab: int = 32768):
    return dict(QWEN3_0_6B, hidden_size=width, intermediate_size=3 * width, num_hidden_layers=layers,
                num_attention_heads=width // 128 * 2, num_key_value_heads=width // 128, head_dim=128, vocab_size=vocab,
                tie_word_embeddings=False, bos_token_id=1, eos_token_id=2)


def _build(raw):
    import torch
    from pih_b200.config import config_from_dict
    from pih_b200.kernels import get_ops
    from pih_b200.models import CausalLM, expected_tensors
    from pih_b200.parts import Runtime
    from pih_b200.weights import random_tensors
    spec = config_from_dict(raw).model_spec()
    dev = torch.device("cuda:0")
    weights = random_tensors(expected_tensors(spec), seed=2, sigma=0.02, dtype=torch.bfloat16)
    return CausalLM(spec, weights, Runtime(dev, torch.bfloat16, get_ops(dev)))


def _timed_steps(model, batch: int, context: int, prompt: int, steps: int):
    """(ms of one prompt of ``prompt`` tokens in one step, ms of a decode step of ``batch`` requests holding ``context``
    tokens each), device-timed, medians; the requests' contexts are run through the model so that states and caches
    hold what the model wrote."""
    import torch
    from pih_b200.engine import StepEntry
    from pih_b200.engine.factory import runner_for
    rt = model.rt
    g = torch.Generator().manual_seed(5)
    cache, runner = runner_for(model, page_size=PAGE, max_cache_tokens=batch * (context + 2 * steps + 64) + prompt + 64,
                               max_requests=batch + 1, cuda_graphs=True, capture_decode_after=2)

    def timed(fn):
        torch.cuda.synchronize()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        return a.elapsed_time(b)

    toks = torch.randint(0, model.spec.vocab, (prompt,), generator=g).tolist()
    pre = []
    for i in range(6):
        pre.append(timed(lambda: runner.step([StepEntry("p", toks, [prompt - 1])])))
        runner.finish("p")
    for r in range(batch):
        runner.step([StepEntry(r, torch.randint(0, model.spec.vocab, (context,), generator=g).tolist(), [])])
    tokens = torch.randint(0, model.spec.vocab, (batch,), generator=g).tolist()

    def decode():
        for _ in range(steps):
            rt.ops.argmax(runner.step([StepEntry(r, [tokens[r]], [0]) for r in range(batch)]))

    decode()                                               # (captures the decode shape)
    dec = sorted(timed(decode) / steps for _ in range(3))[1]
    rt.ops.check_errors()
    for r in range(batch):
        runner.finish(r)
    return sorted(pre[2:])[len(pre[2:]) // 2], dec


def _graph_us(fn, sets, calls: int = 24, repeats: int = 5) -> float:
    """Microseconds of one call as a step sees it: ``calls`` calls in a row on ``sets`` different inputs inside one CUDA
    graph, device-timed, median of ``repeats`` replays."""
    import torch
    for i in range(sets):
        fn(i)
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        for c in range(calls):
            fn(c % sets)
    graph.replay()
    times = []
    for _ in range(repeats):
        torch.cuda.synchronize()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        graph.replay()
        b.record()
        torch.cuda.synchronize()
        times.append(a.elapsed_time(b) / calls * 1e3)
    return sorted(times)[len(times) // 2]


def _step_for_kernels(decode: bool, batch: int, prompt: int, context: int):
    """(what the kernels want to know of a step, its rows, its requests): one prompt, or a decoded token of each of
    ``batch`` requests behind ``context - 1`` others."""
    import types
    import torch
    counts = [1] * batch if decode else [prompt]
    starts = [context - 1] * batch if decode else [0]
    cu = [0]
    for c in counts:
        cu.append(cu[-1] + c)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda:0")
    return types.SimpleNamespace(
        num_requests=len(counts), cu_q=i32(cu), q_start=i32(starts), state_slots=i32(range(len(counts))),
        host_cu_q=cu, host_q_start=starts, attention_plans={}, meta=None,
        request_of_row=i32([r for r, c in enumerate(counts) for _ in range(c)]),
        positions=i32([starts[r] + i for r, c in enumerate(counts) for i in range(c)])), cu[-1], len(counts)


def _bipulorn_kernels(width: int, batch: int, prompt: int, context: int):
    """The kernels of the Bipulorn design beside the like kernel of another design, as ``_kedavik_kernels``."""
    import torch
    from pih_b200.kernels import get_ops
    ops = get_ops(torch.device("cuda:0"))
    hbm = peaks()[0]
    dev, bf, f32 = "cuda:0", torch.bfloat16, torch.float32
    H, d, inner, N = width // 128, 128, 2 * width, 128
    rows_out = []
    for decode in (False, True):
        step, T, R = _step_for_kernels(decode, batch, prompt, context)
        sets = 24 if decode else 6
        rnd = lambda *shape, dtype=bf: [torch.randn(*shape, device=dev, dtype=dtype) for _ in range(sets)]
        vec = lambda n: torch.randn(n, device=dev)

        def add(name, us, nbytes):
            rows_out.append({"kernel": name, "width": width, "step": f"decode x{batch}" if decode else f"prompt {prompt}",
                             "us": round(us, 2), "MB": round(nbytes / 1e6, 2),
                             "of_copy_peak": round(nbytes / (us * 1e-6) / (hbm * 1e9), 4)})

        # the recurrences: q, k, v in, the read-outs out, the states in and out
        qkv, gates, z = rnd(T, 3 * H * d), rnd(T, 2 * H), rnd(T, H * d, dtype=f32)
        moved = T * H * d * (6 + 4) + 2 * R * H * d * d * 4
        cut = lambda i: (qkv[i][:, :H * d], qkv[i][:, H * d:2 * H * d], qkv[i][:, 2 * H * d:])
        kw = dict(step=step, heads=H, key_dim=d, value_dim=d)
        st = rnd(R, H * d * d, dtype=f32)
        bias, dm1 = vec(H * d), -torch.rand(H, device=dev) * 0.03
        for chunked in (True, False) if not decode else (True,):
            ops.chunked_memory = chunked
            how = "" if chunked else ", token by token"
            add("gated_linear" + how, _graph_us(lambda i: ops.gated_linear(*cut(i), z[i], bias=bias, temperature=16.0,
                                                                          q_scale=d ** -0.5, state=st[i], **kw), sets), moved + T * H * d * 4)
            sm = rnd(R, H * (d * d + d + ops.memory_copies(d)), dtype=f32)
            b = vec(H)
            add("matrix_memory" + how, _graph_us(lambda i: ops.matrix_memory(
                *cut(i), gates[i][:, :H], gates[i][:, H:], write_bias=b, keep_bias=b, cap=15.0, floor=1e-6, q_scale=d ** -0.5,
                state=sm[i], **kw), sets), moved + T * H * 8)
            heads = inner // 64
            xbc, dt, ss = rnd(T, inner + 2 * N), rnd(T, heads), rnd(R, heads * N * 64, dtype=f32)
            A, bh = -torch.rand(heads, device=dev), vec(heads)
            add("state_space" + how, _graph_us(lambda i: ops.state_space(
                xbc[i][:, inner + N:], xbc[i][:, inner:inner + N], xbc[i][:, :inner], dt[i], dt_bias=bh, A=A, D=bh, state=ss[i],
                step=step, heads=heads, groups=1, state_dim=N, value_dim=64), sets),
                T * (inner * (2 + 4) + 4 * N + 2 * heads) + 2 * R * heads * N * 64 * 4)
            del sm, xbc, dt, ss
        ops.chunked_memory = True
        add("retention (Tuganex)", _graph_us(lambda i: ops.retention(qkv[i][:, :2 * H * d], qkv[i][:, 2 * H * d:], frequencies=None,
                                                                     decay_minus_one=dm1, key_scale=d ** -0.5, state=st[i], **kw), sets), moved)
        del qkv, gates, z, st
        # the attention with a gate a column beside the one with a gate a head, and what prepares its rows
        G, pages, span = max(1, H // 2), -(-context // PAGE), 1024
        tables = torch.arange(R * pages, dtype=torch.int32, device=dev).view(R, pages)
        cache, src, gate = rnd(R * pages, PAGE, 2 * G * d), rnd(T, (H + 2 * G) * d), rnd(T, H * d)
        geo = dict(heads=H, kv_heads=G, key_dim=d, value_dim=d)
        common = dict(block_table=tables, step=step, scale=d ** -0.5, keep_first=0, softcap=0.0, bias=None, window=span, sink=None, **geo)
        seen = R * span if decode else prompt
        nbytes = T * H * d * 4 + seen * 2 * G * d * 2
        q = [s_[:, :H * d].contiguous() for s_ in src]
        add(f"window_attention, window of {span}, gate a column",
            _graph_us(lambda i: ops.window_attention(q[i], cache=cache[i], gate=gate[i], gate_per="column", **common), sets), nbytes + T * H * d * 2)
        add(f"window_attention, window of {span}, gate a head (Kedavik)",
            _graph_us(lambda i: ops.window_attention(q[i], cache=cache[i], gate=gate[i], **common), sets), nbytes)
        slots = (torch.arange(R, dtype=torch.int32, device=dev).repeat_interleave(T // R) * pages * PAGE
                 + torch.arange(T, dtype=torch.int32, device=dev) % (T // R)).to(torch.int32)
        freq, b_in = torch.rand(32, device=dev), vec((H + 2 * G) * d)
        prep = dict(q_norm=None, k_norm=None, eps=0.0, rope_table=None, rotary_dim=64, positions=step.positions, slot_mapping=slots,
                    values_from_keys=False, frequencies=freq, **geo)
        for name, extra in (("window_qk_prepare, biases, neighbouring pairs", dict(interleaved=True, in_bias=b_in)),
                            ("window_qk_prepare, halves (Kedavik)", dict(interleaved=False))):
            add(name, _graph_us(lambda i: ops.window_qk_prepare(src[i], cache=cache[i], **prep, **extra), sets), T * (H + 2 * G) * d * 4)
        del cache, src, gate, q
        # the norms
        y, gz, wv = rnd(T, inner, dtype=f32), rnd(T, inner), vec(inner)
        add("gated_part_rmsnorm", _graph_us(lambda i: ops.gated_part_rmsnorm(y[i], gz[i], wv, 1, 1e-6), sets), T * inner * 8)
        add("gated_rmsnorm (Rigotar)", _graph_us(lambda i: ops.gated_rmsnorm(y[i].view(T, -1, d), gz[i], wv[:d], 1e-6), sets), T * inner * 8)
        del y, gz
        h, a, b2 = rnd(T, width, dtype=f32), rnd(T, width), rnd(T, width)
        w1 = vec(width)
        add("stream_norm_norm", _graph_us(lambda i: ops.stream_norm_norm(h[i], a[i], w1, 1e-6, w1, 1e-6), sets), T * width * 12)
        add("stream_norm_norm, a pair", _graph_us(lambda i: ops.stream_norm_norm(h[i], a[i], w1, 1e-6, w1, 1e-6, bias=w1,
                                                                                pair=(b2[i], None, w1, w1, 1e-6)), sets), T * width * 14)
        add("rmsnorm_stream (Rigotar)", _graph_us(lambda i: ops.rmsnorm_stream(h[i], w1, 1e-6, delta=a[i]), sets), T * width * 12)
        add("stream_norm_add (Tuganex)", _graph_us(lambda i: ops.stream_norm_add(h[i], a[i], w1, 1e-6, copy_dtype=bf), sets), T * width * 12)
        del h, a, b2
        torch.cuda.empty_cache()
    ops.check_errors()
    return rows_out


def _kedavik_kernels(width: int, batch: int, prompt: int, context: int):
    """The kernels of the Kedavik design beside the like kernel of another design, one prompt of ``prompt`` tokens and one
    decode step of ``batch`` requests: microseconds a call, the bytes that it has to move, and the fraction of the
    measured copy bandwidth that this makes.  Several sets of inputs and states in turn, together larger than L2."""
    import torch
    from pih_b200.kernels import get_ops
    ops = get_ops(torch.device("cuda:0"))
    hbm = peaks()[0]
    dev, bf, f32 = "cuda:0", torch.bfloat16, torch.float32
    heads, d, n, inner, group = width // 128, 128, 16, 2 * width, 2
    rows_out = []

    for decode in (False, True):
        step, T, R = _step_for_kernels(decode, batch, prompt, context)
        sets = 24 if decode else 6
        rnd = lambda *shape, dtype=bf: [torch.randn(*shape, device=dev, dtype=dtype) for _ in range(sets)]

        def add(name, us, nbytes):
            rows_out.append({"kernel": name, "width": width, "step": f"decode x{batch}" if decode else f"prompt {prompt}",
                             "us": round(us, 2), "MB": round(nbytes / 1e6, 2),
                             "of_copy_peak": round(nbytes / (us * 1e-6) / (hbm * 1e9), 4)})

        # the scan beside the other diagonal recurrence (both with what makes their coefficients)
        u, dt, bc, z = rnd(T, inner), rnd(T, inner, dtype=f32), rnd(T, 2 * n), rnd(T, inner)
        st = rnd(R, inner * n, dtype=f32)
        A, vec = -torch.rand(inner, n, device=dev), torch.randn(inner, device=dev)
        add("selective_scan", _graph_us(lambda i: ops.selective_scan(u[i], dt[i], bc[i], z[i], dt_bias=vec, A=A, D=vec, state=st[i],
                                                                     step=step), sets),
            T * (inner * (2 + 4 + 2 + 2) + 4 * n) + (2 * R + 1) * inner * n * 4)
        del u, dt, bc, z, st
        W = width
        u, gates, y, st = rnd(T, W), rnd(T, heads, 2 * W // heads, dtype=f32), rnd(T, W), rnd(R, W, dtype=f32)
        v = torch.randn(W, device=dev)
        add("rglru_scan (Rigotar)", _graph_us(lambda i: ops.rglru_scan(u[i], gates[i], y[i], y_bias=v, r_bias=v, i_bias=v, lam=v,
                                                                       decay_scale=8.0, state=st[i], step=step, blocks=heads), sets),
            T * W * (2 + 8 + 2 + 2) + 2 * R * W * 4)
        del u, gates, y, st
        # the delta rule with a decay a key channel beside the one with a decay a head
        G = max(1, heads // group)
        qkv, b, st = rnd(T, (2 * G + heads) * d), rnd(T, heads), rnd(R, heads * d * d, dtype=f32)
        log, fixed = torch.zeros(heads, device=dev), T * ((2 * G + heads) * d * 2 + heads * 2 + heads * d * 4) + 2 * R * heads * d * d * 4
        kw = dict(decay_log=log, step=step, heads=heads, kv_heads=G, key_dim=d, value_dim=d, unit_eps=1e-6, q_scale=d ** -0.5)
        a, bias = rnd(T, heads * d, dtype=f32), torch.randn(heads * d, device=dev)
        add("gated_delta_rule, decay a channel",
            _graph_us(lambda i: ops.gated_delta_rule(qkv[i], b[i], a[i], decay_bias=bias, state=st[i], **kw), sets),
            fixed + T * heads * d * 4)
        a, bias = rnd(T, heads), torch.randn(heads, device=dev)
        add("gated_delta_rule, decay a head (Rigotar)",
            _graph_us(lambda i: ops.gated_delta_rule(qkv[i], b[i], a[i], decay_bias=bias, state=st[i], **kw), sets),
            fixed + T * heads * 2)
        del qkv, b, st, a
        # attention inside chunks beside the same attention over a window of as many keys
        pages = -(-context // PAGE)
        tables = torch.arange(R * pages, dtype=torch.int32, device=dev).view(R, pages)
        q, cache, gate = rnd(T, heads * d), rnd(R * pages, PAGE, 2 * G * d), rnd(T, heads)
        sink = torch.zeros(heads, device=dev)
        span = 1024
        common = dict(block_table=tables, step=step, scale=d ** -0.5, keep_first=0, softcap=0.0, bias=None, heads=heads,
                      kv_heads=G, key_dim=d, value_dim=d)
        seen = R * span if decode else prompt
        nbytes = T * heads * d * 4 + seen * 2 * G * d * 2
        add(f"window_attention, chunks of {span}, gate a head",
            _graph_us(lambda i: ops.window_attention(q[i], cache=cache[i], window=0, chunk=span, sink=None, gate=gate[i], **common), sets),
            nbytes)
        add(f"window_attention, window of {span}, sink (Sagelorn)",
            _graph_us(lambda i: ops.window_attention(q[i], cache=cache[i], window=span, sink=sink, gate=None, **common), sets),
            nbytes)
        del q, cache, gate
        # the norm of the stream with everything that a pass of the loop adds, beside the plain one; the two activations
        h, y = rnd(T, width, dtype=f32), rnd(T, width)
        table, ids = torch.randn(32768, width, device=dev, dtype=bf), torch.randint(0, 32768, (T,), dtype=torch.int32, device=dev)
        wv = torch.randn(width, device=dev)
        add("rmsnorm_stream, factor, bias, embedding, vector",
            _graph_us(lambda i: ops.rmsnorm_stream(h[i], wv, 1e-6, delta=y[i], scale=0.4, bias=wv, again=(table, ids, 0.5), vector=wv), sets),
            T * width * (8 + 2 + 2 + 2))
        add("rmsnorm_stream (Rigotar)", _graph_us(lambda i: ops.rmsnorm_stream(h[i], wv, 1e-6, delta=y[i]), sets), T * width * (8 + 2 + 2))
        zz, bz = rnd(T, 4 * width), torch.randn(4 * width, device=dev)
        add("activation gelu_erf with bias", _graph_us(lambda i: ops.activation(zz[i], "gelu_erf", bz), sets), T * 16 * width)
        add("bias_xielu (Tuganex)", _graph_us(lambda i: ops.bias_xielu(zz[i], bz, 0.8, 0.8), sets), T * 16 * width)
        del h, y, zz
        torch.cuda.empty_cache()
    ops.check_errors()
    return rows_out


def design_run(args) -> int:
    """``--design rigotar``: prompt and decode throughput of the Rigotar design at two widths with layer sizes that
    resemble a real model's (random weights, bf16), beside the dense decoder at the same width, depth and number of
    active feed-forward weights; and every mixer alone (four layers of it, no feed-forward) beside the dense model's
    attention-only time, so that each kind of layer can be read off.  One JSON line."""
    import torch
    rows = []
    batch, context, prompt, steps = args.batch, CONTEXT, PREFILL_TOKENS, max(8, args.steps // 4)
    with ClockSampler() as clocks:
        for width in (1024, 2048):
            if args.design == "bipulorn":
                # the design beside the models nearest to it (a matrix state with a fixed decay and the same experts; two mixers
                # side by side) and the dense decoder; and each of its kinds of layer alone beside its like
                cases = [("bipulorn", _bipulorn_config(width, 8)), ("tuganex", _tuganex_config(width, 8, mlps=("moe",))),
                         ("kedavik", _kedavik_config(width, 8)), ("dense", _dense_config(width, 8))]
                if width == 1024:
                    cases += [(f"bipulorn {k} x4, no feed-forward", _bipulorn_config(width, 4, kinds=(k,), moe=False))
                              for k in ("gla", "mlstm", "parallel")]
                    cases += [("tuganex retention x4, no feed-forward", _tuganex_config(width, 4, kinds=("retention",), mlps=None)),
                              ("kedavik parallel x4, no feed-forward", _kedavik_config(width, 4, kinds=("parallel",), mlp=False)),
                              ("bipulorn gla x4 with experts", _bipulorn_config(width, 4, kinds=("gla",))),
                              ("tuganex retention x4 with experts", _tuganex_config(width, 4, kinds=("retention",), mlps=("moe",)))]
            elif args.design == "kedavik":
                # the design beside the model nearest to it (a diagonal recurrence, a delta rule, attention) and the dense
                # decoder; and each of its kinds of layer alone beside its like
                cases = [("kedavik", _kedavik_config(width, 8)), ("rigotar", _rigotar_config(width, 8)),
                         ("dense", _dense_config(width, 8))]
                if width == 1024:
                    cases += [(f"kedavik {k} x4, no feed-forward", _kedavik_config(width, 4, kinds=(k,), mlp=False))
                              for k in ("mamba1", "parallel")]
                    cases += [("rigotar rglru x4, no feed-forward", _rigotar_config(width, 4, kinds=("rglru",), moe=False)),
                              ("rigotar delta x4, no feed-forward", _rigotar_config(width, 4, kinds=("delta",), moe=False)),
                              ("sagelorn attention x4, no feed-forward",
                               _sagelorn_config(width, 4, kinds=("attention",), mlps=None, share=False)),
                              ("kedavik parallel x4, dense feed-forward", _kedavik_config(width, 4, kinds=("parallel",))),
                              ("tuganex retention x4, no feed-forward", _tuganex_config(width, 4, kinds=("retention",), mlps=None)),
                              ("tuganex retention x4, dense feed-forward",
                               _tuganex_config(width, 4, kinds=("retention",), mlps=("dense",))),
                              ("kedavik 2 layers run 4 times", _kedavik_config(width, 4, loop=(1, 3, 4)))]
            elif args.design == "sagelorn":
                # the design beside the model nearest to it (norms on the outputs, retention, shared caches, routed experts
                # with a shared one) and the dense decoder; and each of its kinds of layer alone beside its like
                cases = [("sagelorn", _sagelorn_config(width, 8)), ("tuganex", _tuganex_config(width, 8, share_from=6)),
                         ("dense", _dense_config(width, 8))]
                if width == 1024:
                    cases += [(f"sagelorn {k} x4, no feed-forward", _sagelorn_config(width, 4, kinds=(k,), mlps=None, share=False))
                              for k in ("attention", "latent_attention", "retention")]
                    cases += [("sagelorn attention x4, every second reads the one before", _sagelorn_config(width, 4, kinds=("attention",), mlps=None)),
                              ("pegopel attention_2 x4, no feed-forward, one stream",
                               _pegopel_config(width, 4, kinds=("attention_2",), mlp=False, streams=0)),
                              ("rigotar latent_attention x4, no feed-forward", _rigotar_config(width, 4, kinds=("latent_attention",), moe=False)),
                              ("tuganex retention x4, no feed-forward", _tuganex_config(width, 4, kinds=("retention",), mlps=None)),
                              ("sagelorn retention x4 with experts", _sagelorn_config(width, 4, kinds=("retention",), mlps=("moe",))),
                              ("tuganex retention x4 with experts", _tuganex_config(width, 4, kinds=("retention",), mlps=("moe",))),
                              ("sagelorn retention x4, dense feed-forward", _sagelorn_config(width, 4, kinds=("retention",), mlps=("dense",))),
                              ("tuganex retention x4, dense feed-forward", _tuganex_config(width, 4, kinds=("retention",), mlps=("dense",)))]
            elif args.design == "pegopel":
                # the design beside the models nearest to it (softmax attention over pages and a gated dense
                # feed-forward), and each of its mixers alone, seeing every key, beside the other attentions alone
                cases = [("pegopel", _pegopel_config(width, 8)), ("pegopel, every key seen", _pegopel_config(width, 8, window=8192)),
                         ("dense", _dense_config(width, 8)),
                         ("tuganex attention, dense feed-forward", _tuganex_config(width, 8, kinds=("attention",), mlps=("dense",)))]
                if width == 1024:
                    cases += [(f"pegopel {k} x4, no feed-forward, every key seen",
                               _pegopel_config(width, 4, kinds=(k,), window=8192, mlp=False)) for k in ("attention", "attention_2")]
                    cases += [(f"pegopel {k} x4, no feed-forward", _pegopel_config(width, 4, kinds=(k,), mlp=False))
                              for k in ("attention", "attention_2")]
                    cases += [("tuganex attention x4, no feed-forward", _tuganex_config(width, 4, kinds=("attention",), mlps=None)),
                              ("pegopel attention x4, one stream", _pegopel_config(width, 4, kinds=("attention",), streams=0)),
                              ("pegopel 2 layers run 4 times", _pegopel_config(width, 4, loop=(1, 3, 4)))]
            elif args.design == "tuganex":
                # the design beside the two models that are nearest to it (mixers with a state and routed experts; a
                # softmax attention and a dense feed-forward), and each of its kinds of layer alone beside its like
                cases = [("tuganex", _tuganex_config(width, 8, share_from=6)), ("rigotar", _rigotar_config(width, 8)),
                         ("dense", _dense_config(width, 8))]
                if width == 1024:
                    cases += [(f"tuganex {k} x4, no feed-forward", _tuganex_config(width, 4, kinds=(k,), mlps=None))
                              for k in ("retention", "attention")]
                    cases += [("rigotar delta x4, no feed-forward", _rigotar_config(width, 4, kinds=("delta",), moe=False)),
                              ("tuganex retention x4, dense feed-forward", _tuganex_config(width, 4, kinds=("retention",), mlps=("dense",))),
                              ("tuganex retention x4 with experts", _tuganex_config(width, 4, kinds=("retention",), mlps=("moe",))),
                              ("rigotar delta x4 with experts", _rigotar_config(width, 4, kinds=("delta",)))]
            else:
                cases = [("rigotar", _rigotar_config(width, 8)), ("dense", _dense_config(width, 8))]
                if width == 1024:
                    cases += [(f"rigotar {k} x4, no feed-forward", _rigotar_config(width, 4, kinds=(k,), moe=False))
                              for k in ("rglru", "latent_attention", "delta")]
                    cases += [("rigotar rglru x4 with experts", _rigotar_config(width, 4, kinds=("rglru",)))]
            for name, raw in cases:
                model = _build(raw)
                pre_ms, dec_ms = _timed_steps(model, batch, context, prompt, steps)
                rows.append({"model": name, "width": width, "layers": len(raw.get("layers", [])) or raw["num_hidden_layers"],
                             "prefill_ms": round(pre_ms, 3), "prefill_tok_s": round(prompt / pre_ms * 1e3),
                             "decode_ms": round(dec_ms, 4), "decode_tok_s": round(batch / dec_ms * 1e3)})
                del model
                gc.collect()
                torch.cuda.empty_cache()
        alone = {"kedavik": _kedavik_kernels, "bipulorn": _bipulorn_kernels}.get(args.design)
        kernels = {"kernels": alone(1024, batch, prompt, context)} if alone is not None else {}
        clock_summary = clocks.summary()
    print(json.dumps({"metric": f"prompt and decode tok/s of the {args.design.capitalize()} design beside the framework's other models",
                      "dtype": "bf16",
                      "data": "synthetic", "n_gpus": 1, "config": {"prompt_tokens": prompt, "decode_batch": batch,
                                                                   "context": context, "page_size": PAGE},
                      "rows": rows, **kernels, "clocks": clock_summary}))
    return 0


def reference_arm():
    print(json.dumps({"impl": "reference", "unavailable":
                      "pip installs only pih_client, an HTTP client; the engine is a C++20/CUDA worker (CMake) whose "
                      "kernels are built as sm_89/sm_90 cubins only, which a B200 (sm_100) cannot load, and which "
                      "its own docs call unverified on any GPU"}))
    return 0


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--layers", type=int, default=28)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--skip-e2e", action="store_true")
    ap.add_argument("--skip-points", action="store_true")
    ap.add_argument("--skip-prefill", action="store_true")
    ap.add_argument("--design", default=None, choices=["rigotar", "tuganex", "pegopel", "sagelorn", "kedavik", "bipulorn"],
                    help="instead of the recorded workload: this design's prompt and decode throughput beside the dense decoder's")
    ap.add_argument("--plain-launches", action="store_true",
                    help="launch kernels fully serialised instead of with programmatic dependent launch")
    args = ap.parse_args()
    if args.impl == "reference":
        return reference_arm()
    if args.gpus != 1:
        print(f"bench.py: this engine runs on one GPU; --gpus {args.gpus} is not supported")
        return 2
    if args.warmup < 3:
        args.warmup = 3

    if args.design is not None:
        return design_run(args)

    import torch
    hbm_gbs, bf16_tflops, peak_src = peaks()
    config, model = build_model(args.layers)
    if args.plain_launches:
        model.rt.ops.set_dependent_launch(False)
    with ClockSampler() as clocks:
        main_run = decode_run(model, args.batch, args.steps, args.warmup)
        clock_summary = clocks.summary()
    # the end-to-end number directly after the device-timed one, with its own clock record: measured after the
    # batch-64 and prompt runs below it came out 6 % lower (1.21 against 1.15 ms a step) with nothing else changed
    e2e = None
    if not args.skip_e2e:
        from pih_b200.weights import write_random_model
        with tempfile.TemporaryDirectory() as d:
            write_random_model(d, config, seed=2, sigma=0.02)
            with ClockSampler() as clocks:
                e2e = e2e_run(config, d, args.batch, args.steps, args.warmup)
                e2e["sm_mhz"] = clocks.summary()["sm_mhz"]
        torch.cuda.empty_cache()
    points = {}
    if not args.skip_points:
        for b in (1, 64):
            points[f"decode_b{b}"] = round(decode_run(model, b, max(8, args.steps // 2), 3, repeats=3)["tok_s"], 1)
    pre = None if args.skip_prefill else prefill_run(model, PREFILL_TOKENS)
    achieved = main_run["bytes"] / (main_run["ms"] * 1e-3) / 1e9
    line = {
        "metric": METRIC.replace("batch 8", f"batch {args.batch}"), "value": round(main_run["tok_s"], 1), "unit": "tok/s", "n_gpus": 1,
        "steps": args.steps, "warmup": args.warmup, "ms_per_step": round(main_run["ms"], 4),
        "timed_loops_ms_per_step": main_run["loops_ms"],
        "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
        "impl": "ours",
        "config": {"model": "Qwen3-0.6B random weights seed 2", "layers": args.layers, "layers_of_config": 28,
                   "hidden": config.hidden_size, "heads": config.num_attention_heads,
                   "kv_heads": config.num_key_value_heads, "head_dim": config.head_dim,
                   "intermediate": config.intermediate_size, "vocab": config.vocab_size,
                   "tied_embeddings": config.tie_word_embeddings, "global_batch": args.batch, "seq_len": CONTEXT,
                   "context_window": 4096, "page_size": PAGE, "prefill_tokens": PREFILL_TOKENS,
                   "parallelism": "single GPU", "l2": "inputs larger than L2", "peaks": peak_src},
        "e2e": e2e,
        "gpu_launches": main_run["launches"],
        "clocks": clock_summary,
        "prefill": None if args.skip_prefill else {
            "value": round(pre["tok_s"], 1), "tokens": PREFILL_TOKENS, "ms": round(pre["ms"], 3),
            "frac": round(pre["flops"] / (pre["ms"] * 1e-3) / (bf16_tflops * 1e12), 4),
            "first_sight_ms": round(pre["first_sight_ms"], 3)},
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": hbm_gbs, "unit": "GB/s",
                     "frac": round(achieved / hbm_gbs, 4)},
        "points": points,
    }
    print(json.dumps(line))
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
