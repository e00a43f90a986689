#!/usr/bin/env python3
"""Benchmark of the engine's decode step on one B200: ``python bench.py --gpus 1 --steps K --warmup W``.

The model has the layer sizes of the MiniCPM-2B shape (40 layers, hidden 2304, 36/36 heads of
64, intermediate 5760, vocabulary 122753, tied embeddings) with random bfloat16 weights made
on the device.  A step is one decode step of a batch of 8 requests whose caches hold about
4096 tokens each (synthetic cache contents: decoding cost does not depend on the values).

One JSON line is printed:
  value       decoded tokens per second, device-timed (CUDA events around K steps of the engine's
              step function + the sampling kernel; token ids are fixed, nothing is read back);
  e2e         the same through the Python entry point (``batch_infer_one_round``): every step copies
              its token ids and block tables from pinned host memory and reads the sampled ids back;
  prefill     one 2,048-token prompt through the step function;
  roofline    bytes a decode step must read (every weight once + the live requests' cache) / time;
  points      decode tokens per second at batch 1 and 64 (context 4096) and at context 512;
  plain       the same engine run one call per operator with library products, the plain attention kernel, separate norm
              kernels and no CUDA graphs: the shape of the reference's step (src/models/jiuge/jiuge.cpp:195-258), which
              cannot itself be built here; ``vs_baseline`` is ``value`` over this path's batch-8 decode rate;
  kernels     device time of each dominant kernel alone at the benchmark's shape (one launch record of the model at a time,
              walking through the layers so that weights and cache come from memory, not from L2) with its achieved
              GB/s or TFLOP/s over the measured peak.
Peaks come from MEASURED_PEAKS.json beside this file if present, else from the fallback values.
"""
import argparse
import json
import os
import statistics
import subprocess
import sys
import tempfile
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

# configs[2] of the benchmark definition: the MiniCPM-2B shape
SHAPE_2B = dict(model_type="minicpm", num_hidden_layers=40, hidden_size=2304, num_attention_heads=36,
                num_key_value_heads=36, intermediate_size=5760, vocab_size=122753,
                max_position_embeddings=4096, rms_norm_eps=1e-5, rope_theta=10000.0, scale_emb=12,
                scale_depth=1.4, dim_model_base=256, tie_word_embeddings=True)
# the shapes of the two serving-style workloads (--workload)
SHAPE_1B = dict(model_type="minicpm", num_hidden_layers=52, hidden_size=1536, num_attention_heads=24,
                num_key_value_heads=8, intermediate_size=3840, vocab_size=73440,
                max_position_embeddings=4096, rms_norm_eps=1e-5, rope_theta=10000.0, scale_emb=12,
                scale_depth=1.4, dim_model_base=256, tie_word_embeddings=True)
SHAPE_8B = dict(model_type="fm9g", num_hidden_layers=32, hidden_size=4096, num_attention_heads=32,
                num_key_value_heads=2, intermediate_size=16384, vocab_size=73448,
                max_position_embeddings=4096, rms_norm_eps=1e-5, rope_theta=10000.0, scale_emb=12,
                scale_depth=1.4, dim_model_base=256, tie_word_embeddings=False)
WORKLOADS = {
    # name: (shape, requests, prompt lengths, new tokens, portion size, token budget of a step)
    "1b-mixed": (SHAPE_1B, 32, (16, 1024), 128, 256, 512),
    "8b-serving": (SHAPE_8B, 64, (512, 2048), 256, 512, 2048),
}
FALLBACK_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0}


def load_peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.isfile(path):
        try:
            with open(path) as f:
                data = json.load(f)
            flat = {}
            def walk(d):
                for k, v in d.items():
                    if isinstance(v, dict):
                        walk(v)
                    elif isinstance(v, (int, float)):
                        flat.setdefault(k, float(v))
            walk(data)
            if "hbm_gbs" in flat and "bf16_tflops" in flat:
                return {"hbm_gbs": flat["hbm_gbs"], "bf16_tflops": flat["bf16_tflops"],
                        "bf16_tflops_sustained": flat.get("bf16_tflops_sustained", flat["bf16_tflops"])}, "measured"
        except (OSError, ValueError):
            pass
    return dict(FALLBACK_PEAKS), "fallback"


class ClockSampler:
    """nvidia-smi in the background while the timed region runs; stopped by its own PID."""
    QUERY = ("clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.active,"
             "clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __enter__(self):
        self.file = tempfile.NamedTemporaryFile("w+", suffix=".csv", delete=False)
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", "-i", "0", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits", "-lms", "100"],
                stdout=self.file, stderr=subprocess.DEVNULL)
        except OSError:
            self.proc = None
        return self

    def __exit__(self, *exc):
        if self.proc is not None:
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()
        self.file.flush()

    def summary(self):
        self.file.seek(0)
        sm, mx, reasons = [], [], set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for line in self.file.read().splitlines():
            parts = [p.strip() for p in line.split(",")]
            if len(parts) < 8:
                continue
            try:
                sm.append(float(parts[0])); mx.append(float(parts[1]))
            except ValueError:
                continue
            for name, val in zip(names, parts[4:8]):
                if val.lower().startswith("active"):
                    reasons.add(name)
        self.file.close()
        os.unlink(self.file.name)
        if not sm:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["no samples"]}
        return {"sm_mhz": statistics.median(sm), "sm_max_mhz": max(mx), "reasons": sorted(reasons), "samples": len(sm)}


def run_workload(name, layers=None):
    """A serving-style workload through the scheduler: all requests are submitted at once, prompts are
    cut into portions under the step's token budget beside the others' decoded tokens, every request
    generates its full count (no stop token).  Prints one JSON line of its own kind."""
    import random
    import torch
    from infinicore_infer_b200.config import MiniCPMConfig
    from infinicore_infer_b200.engine import Engine, Generator
    from infinicore_infer_b200.parts import model_manifest
    from infinicore_infer_b200.weights import DeviceRandomWeights

    shape, n_req, (lo, hi), new_tokens, chunk, budget = WORKLOADS[name]
    shape = dict(shape)
    full_layers = shape["num_hidden_layers"]
    if layers:
        shape["num_hidden_layers"] = layers
    cfg = MiniCPMConfig.from_dict(shape)
    spec = cfg.model_spec()
    dev, page = "cuda:0", 16
    rng = random.Random(0)
    prompts = [[rng.randrange(cfg.vocab_size) for _ in range(rng.randint(lo, hi))] for _ in range(n_req)]
    cache_tokens = sum(len(p) + new_tokens + page for p in prompts)
    weights = DeviceRandomWeights(model_manifest(spec), seed=0, compute_dtype=torch.bfloat16, device=dev, std=0.02,
                                  untied=not shape["tie_word_embeddings"])
    engine = Engine(spec, weights, dtype=torch.bfloat16, device=dev, cache_tokens=cache_tokens, page_size=page,
                    max_requests=n_req, max_step_tokens=budget)
    results = []
    with ClockSampler() as clocks:
        for rep in range(2):                   # the first pass warms up (graph captures, lazy handles)
            g = Generator(engine, max_batch=n_req, max_tokens_per_step=budget, chunk_size=chunk)
            reqs = [g.submit(p, max_new_tokens=new_tokens, eos_token_ids=()) for p in prompts]
            torch.cuda.synchronize()
            l0 = engine.kernel_launches
            t0 = time.perf_counter()
            g.run()
            torch.cuda.synchronize()
            dt = time.perf_counter() - t0
            generated = sum(len(r.generated) for r in reqs)
            results.append((dt, generated, dict(g.scheduler.counters), engine.kernel_launches - l0))
    dt, generated, counters, launches = results[-1]
    prompt_tokens = sum(len(p) for p in prompts)
    print(json.dumps({
        "workload": name, "metric": "generated tok/s through the scheduler (host tokens in and out every step)",
        "value": round(generated / dt, 1), "unit": "tokens/s", "seconds": round(dt, 3),
        "generated_tokens": generated, "prompt_tokens": prompt_tokens,
        "all_tokens_per_s": round((generated + prompt_tokens) / dt, 1),
        "scheduler": counters, "gpu_launches": int(launches), "dtype": "bf16",
        "data": "synthetic: random-init weights N(0,0.02), uniform random token ids",
        "config": {"model": name, "layers": cfg.num_hidden_layers, "layers_of_shape": full_layers,
                   "hidden": cfg.hidden_size, "heads": cfg.num_attention_heads, "kv_heads": cfg.num_key_value_heads,
                   "head_dim": cfg.head_dim, "intermediate": cfg.intermediate_size, "vocab": cfg.vocab_size,
                   "requests": n_req, "prompt_len_min": lo, "prompt_len_max": hi, "new_tokens": new_tokens,
                   "portion": chunk, "tokens_per_step": budget, "page_size": page},
        "clocks": clocks.summary(),
    }))
    return 0



def time_records(engine, ctx, which, repeats=3):
    """Device time (microseconds per launch) of one kind of launch record, run alone: ``which(l)`` gives the index of
    layer l's record (or None to skip the layer).  The records of all layers run one after the other as one CUDA graph,
    so each launch reads its own layer's weights and cache pages from memory and follows its predecessor as closely as
    in a step; the best of ``repeats`` replays counts."""
    import ctypes
    import torch
    from infinicore_infer_b200 import kernels
    from infinicore_infer_b200.parts.program import SLOT, RunnerStep
    runner, prog = engine.runner, engine.program
    T = ctx.ntok
    logits = torch.empty(max(1, ctx.want_rows.numel()), engine.spec.vocab_size, dtype=torch.float32, device=engine.device)
    runner.buffers.slot[SLOT["logits"]] = logits.data_ptr()
    runner.buffers.bytes[SLOT["logits"]] = logits.numel() * 4
    step = RunnerStep(ntok=T, nreq=ctx.nreq, n_want=ctx.want_rows.numel(), context=ctx.context, tokens=ctx.tokens.data_ptr(),
                      positions=ctx.positions.data_ptr(), row_req=ctx.row_req.data_ptr(), req_start=ctx.req_start.data_ptr(),
                      req_pos=ctx.req_pos.data_ptr(), want_rows=ctx.want_rows.data_ptr(), slot_ids=ctx.slot_ids.data_ptr())
    for g, table in enumerate(ctx.block_tables):
        step.block_tables[g] = table.data_ptr()
    for name, index in prog.lists.items():
        view, n = ctx.lists[name]
        step.lists[index] = view.data_ptr() if view is not None else None
        step.list_n[index] = n
    indices = which if isinstance(which, (list, tuple)) else [i for i in (which(l) for l in range(len(engine.spec.order))) if i is not None]

    def walk():
        stream = kernels._stream()          # asked for at each walk: a capture runs on a stream of its own
        for i in indices:
            rc = runner.lib.jk_runner_run(ctypes.byref(runner.env), prog.ops, i, 1, ctypes.byref(step), ctypes.byref(runner.buffers), 1, stream)
            if rc:
                raise RuntimeError(runner.lib.jk_runner_last_error().decode())
    walk()
    torch.cuda.synchronize()
    # the walk as one CUDA graph: launches follow one another as they do in a step (each starts under the tail of the one
    # before), without the host's time between them
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        walk()
    graph.replay()
    torch.cuda.synchronize()
    best = None
    for _ in range(repeats):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        graph.replay()
        e1.record()
        torch.cuda.synchronize()
        us = e0.elapsed_time(e1) * 1000.0 / len(indices)
        best = us if best is None else min(best, us)
    return best


# ---- --design: another architecture beside the decoder of the same size ------------------------------------------------
# Layer sizes that resemble a real model's: (name, width, feed-forward, heads, key/value heads, head size, vocabulary).
DESIGN_SIZES = {"2k": (2048, 5632, 16, 4, 128, 32000), "4k": (4096, 11008, 32, 8, 128, 32000)}
F32_FMA_TFLOPS = 148 * 128 * 2 * 1.965e9 / 1e12      # nominal float32 rate of the CUDA cores (no measured figure exists)


def sitelorn_shape(width, ff, heads, kv_heads, dim, vocab, window, layers=8):
    """Eight layers in the order lightning, gla, attention, lightning, lightning, gla, attention on layer 2's keys,
    lightning: heads of ``dim`` for keys and values everywhere, a window of ``window``, four taps."""
    mlp = {"kind": "dense", "ff": ff}
    light = {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": dim,
                                            "decay": [1.0 - 2.0 ** (-5 - 3 * h / max(1, heads - 1)) for h in range(heads)]}, "mlp": mlp}
    gla = {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": dim, "tau": 16.0, "rank": 16}, "mlp": mlp}
    att = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "conv": 4, "rot": {"dims": dim // 2, "base": 5e5},
           "scale": dim ** -0.5, "mask": {"size": window}}
    order = [light, gla, {"type": "attention", "mixer": att, "mlp": mlp}, light, light, gla,
             {"type": "attention", "mixer": dict(att, kv_from=2), "mlp": mlp}, light]
    return {"architecture": "Sitelorn", "embedding": {"scale": 1.0}, "norm": {"eps": 1e-5}, "vocab": vocab, "width": width,
            "layers": order[:layers]}


def vunelix_shape(width, ff, heads, dim, vocab):
    """Seven layers, eight layer runs (the second layer runs twice): latent attention with plain heads of ``dim``, rotated
    parts of dim / 2, values of ``dim`` and a latent vector of 4 dim; selective scans of 2 width channels with 16 states; a
    dense feed-forward in the first layer, then eight experts of ff / 4 of which a row takes two, and a shared one."""
    att = {"heads": heads, "dim": dim, "rot_dim": dim // 2, "vdim": dim, "kv_rank": 4 * dim, "scale": (dim + dim // 2) ** -0.5,
           "rot": {"base": 1e4, "dims": dim // 2, "scaling": {"factor": 4.0, "original": 1024, "fast": 32.0, "slow": 1.0}}}
    ssm = {"inner": 2 * width, "state": 16, "dt_rank": width // 16, "conv": 4}
    moe = {"kind": "moe", "router": {"experts": 8, "top": 2}, "expert": {"ff": ff // 4}, "shared": {"ff": ff // 4}}
    lat = lambda mlp: {"type": "latent_attention", "mixer": att, "mlp": mlp}
    scan = {"type": "mamba1", "mixer": ssm, "mlp": moe}
    return {"architecture": "Vunelix", "norm": {"eps": 1e-5}, "vocab": vocab, "width": width, "logit_softcap": 30.0,
            "loop": {"start": 1, "stop": 2, "times": 2},
            "layers": [lat({"kind": "dense", "ff": ff}), lat(moe), scan, lat(moe), lat(moe), scan, lat(moe)]}


def vipovik_shape(width, ff, heads, kv_heads, dim, vocab, window):
    """Six layers, eight layer runs (the second and third layer run twice): in every layer attention with heads of ``dim``
    for keys and values, rotated whole with stretched frequencies, capped scores, a window of ``window`` that keeps its first
    four keys, beside a recurrence with heads of 64 over the whole width and a decay projection of 64; feed-forwards in turn
    dense without a gate and eight clamped experts of ff / 4 of which a row takes two."""
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "softcap": 30.0,
            "mask": {"size": window, "keep_first": 4},
            "rot": {"base": 5e5, "dims": dim, "scaling": {"factor": 4.0, "original": 1024, "fast": 32.0, "slow": 1.0}}}
    mixer = {"left": left, "right": {"heads": width // 64, "dim": 64, "rank": 64}, "left_scale": 0.6, "right_scale": 0.5}
    dense = {"kind": "dense", "ff": ff}
    moe = {"kind": "moe", "router": {"experts": 8, "top": 2}, "expert": {"ff": ff // 4, "limit": 7.0}}
    return {"architecture": "Vipovik", "embedding": {"scale": 1.0}, "norm": {"eps": 1e-5}, "vocab": vocab, "width": width,
            "loop": {"start": 1, "stop": 3, "times": 2},
            "layers": [{"type": "parallel", "mixer": mixer, "mlp": mlp} for mlp in (dense, moe, dense, moe, dense, moe)]}


def fapenex_shape(width, ff, heads, kv_heads, dim, vocab, window):
    """Six layers, eight layer runs (the second and third layer run twice): a gated delta rule with heads of ``dim`` x ``dim``
    behind convolutions of four taps; attention with grouped heads of ``dim``, biases, a norm per head, half of each head
    rotated with stretched frequencies, chunks of ``window`` positions and a sink; latent attention with heads of ``dim``, a
    latent vector of 4 dim, queries through a latent of 3/4 width, a window of ``window``.  Every layer has eight clamped
    experts of ff / 4 of which a row takes two, and a shared one with a gate per row.  Learned positions."""
    moe = {"kind": "moe", "router": {"experts": 8, "top": 2}, "expert": {"ff": ff // 4, "limit": 7.0}, "shared": {"ff": ff // 4, "limit": 7.0}}
    delta = {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "conv": 4}, "mlp": moe}
    att = {"type": "attention", "mlp": moe,
           "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "mask": {"size": window},
                     "rot": {"base": 1e4, "dims": dim // 2, "scaling": {"factor": 4.0, "original": 1024, "fast": 32.0, "slow": 1.0}}}}
    lat = {"type": "latent_attention", "mlp": moe,
           "mixer": {"heads": heads, "dim": dim, "vdim": dim, "kv_rank": 4 * dim, "q_rank": 3 * width // 4, "scale": dim ** -0.5,
                     "mask": {"size": window}}}
    return {"architecture": "Fapenex", "norm": {"eps": 1e-5}, "vocab": vocab, "width": width, "max_positions": 8192, "logit_scale": 1.0,
            "logit_softcap": 30.0, "loop": {"start": 1, "stop": 3, "times": 2}, "layers": [delta, att, lat, lat, delta, att]}


def fupapel_shape(width, ff, heads, kv_heads, dim, vocab, window):
    """Eight layers, mixers and feed-forwards side by side behind a token shift: attention with grouped heads of ``dim``, half of
    each head rotated, chunks of ``window`` positions, a gate per output element; the same behind convolutions of three taps with
    stretched frequencies, a factor and a learned sink per head, one such layer on another's keys and values; latent attention
    with heads of ``dim`` plain and ``dim`` / 2 rotated elements, a latent vector of 4 dim, queries through a latent of 3/4 width.
    Every layer has eight experts of ff / 4 and four identities in three groups, of which a row takes three from two groups."""
    moe = {"kind": "moe", "router": {"experts": 8, "identity": 4, "top": 3, "groups": {"count": 3, "keep": 2}}, "expert": {"ff": ff // 4}}
    heads_of = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "mask": {"size": window}}
    att = {"type": "attention", "mlp": moe, "mixer": dict(heads_of, rot={"base": 1e4, "dims": dim // 2})}
    conv = {"type": "attention_2", "mlp": moe,
            "mixer": dict(heads_of, conv=3, rot={"base": 5e5, "dims": dim, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 1024}})}
    borrows = {"type": "attention_2", "mlp": moe, "mixer": dict(conv["mixer"], kv_from=1)}
    lat = {"type": "latent_attention", "mlp": moe,
           "mixer": {"heads": heads, "dim": dim, "rot_dim": dim // 2, "vdim": dim, "kv_rank": 4 * dim, "q_rank": 3 * width // 4,
                     "scale": (1.5 * dim) ** -0.5, "rot": {"base": 1e6, "dims": dim // 2}}}
    return {"architecture": "Fupapel", "norm": {"eps": 1e-5}, "vocab": vocab, "width": width, "residual_mult": 0.5,
            "layers": [att, conv, lat, lat, att, borrows, lat, att]}


def piratar_shape(width, ff, heads, kv_heads, dim, vocab):
    """Eight layers P P R U P R U P, mixers and feed-forwards side by side: P attention with grouped heads of ``dim`` behind
    convolutions of four taps, rotated whole, a gate per output element, beside retention with heads of ``dim`` x ``dim``; U the same
    with attention keys of dim / 2 and values of ``dim`` and retention heads of dim / 2 x dim; R a real-gated recurrence over the width
    with gates' maps of 256.  A dense feed-forward in the first layer, then eight experts of ff / 4 of which a row takes two, and a
    shared one with a gate per row; pairs of tokens, and token vectors of 256 in every layer."""
    decay = lambda n: [1.0 - 2.0 ** (-5 - 6 * h / max(1, n - 1)) for h in range(n)]
    def both(dk):
        return {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dk, "vdim": dim, "scale": dk ** -0.5, "conv": 4, "rot": {"base": 5e5, "dims": dk}},
                "right": {"heads": heads, "dim": dk, "vdim": dim, "decay": decay(heads), "rot": {"base": 1e4, "dims": dk}}}
    dense = {"kind": "dense", "ff": ff}
    moe = {"kind": "moe", "router": {"experts": 8, "top": 2, "scale": 2.0}, "expert": {"ff": ff // 4}, "shared": {"ff": ff // 4}}
    P, U = ({"type": "parallel", "mixer": both(dk), "mlp": moe} for dk in (dim, dim // 2))
    R = {"type": "rglru", "mixer": {"width": width, "blocks": width // 256, "conv": 4}, "mlp": moe}
    return {"architecture": "Piratar", "norm": {"eps": 1e-5}, "vocab": vocab, "width": width,
            "embedding": {"scale": 1.0, "bigram": {"buckets": 65521, "mul_prev": 31, "mul_cur": 17}}, "token_side": {"dim": 256},
            "layers": [dict(P, mlp=dense), P, R, U, P, R, U, P]}


def decoder_shape(width, ff, heads, kv_heads, dim, vocab, layers=8):
    return dict(model_type="llama", num_hidden_layers=layers, hidden_size=width, num_attention_heads=heads, num_key_value_heads=kv_heads,
                head_dim=dim, intermediate_size=ff, vocab_size=vocab, max_position_embeddings=4096, rms_norm_eps=1e-5,
                rope_theta=10000.0, tie_word_embeddings=False)


def record_cost(op, T, B, context, decode, page_bytes):
    """(bytes a record must move, floating-point operations it must do) for a step of T rows of B requests."""
    from infinicore_infer_b200.parts.program import OP_NAMES
    kind = OP_NAMES.get(op.kind)
    dv = op.v_head_dim or op.head_dim
    if kind in ("linear", "qkv", "residual"):
        rows = T if not op.wanted_rows else B
        return 2 * op.n * op.k + 2 * rows * op.k + 4 * rows * op.n, 2.0 * rows * op.n * op.k
    if kind == "gate_up":
        return 2 * 2 * op.n * op.k + 2 * T * op.k + 2 * T * op.n, 2.0 * T * 2 * op.n * op.k
    if kind == "attention":
        reach = min(context, abs(op.window)) if op.window else context      # a negative window: chunks of that many positions
        keys = B * reach if decode else T       # cached rows that are read at least once
        seen = (B * reach) if decode else sum(min(t + 1, reach) for t in range(T))
        gate = 4 * T * op.heads * (dv if op.gated == 2 else 1) if op.gated else 0
        return keys * op.kv_heads * (op.head_dim + dv) * 2 + 2 * T * op.heads * (op.head_dim + dv) + gate, 2.0 * seen * op.heads * (op.head_dim + dv)
    if kind == "linear_attention":
        state = B * op.heads * op.head_dim * dv * 4 * 2
        return state + 4 * T * op.ld + 2 * T * op.heads * dv, 4.0 * T * op.heads * op.head_dim * dv
    if kind == "conv_qkv":
        return 4 * T * op.ld + 2 * T * (op.heads * op.head_dim + (op.kv_heads * (op.head_dim + dv) if op.has_kv else 0)), 0.0
    if kind == "token_shift":
        return T * op.n * 2 * (1 + op.heads) + B * op.n * 8, 2.0 * T * op.n * op.heads
    if kind == "activate":
        return T * op.n * (4 + 2 + (2 if op.w else 0)), 0.0
    if kind == "rotate":
        return T * op.heads * op.rot_dims * 2 * (4 + 4), 0.0
    if kind == "embed_pair":
        return T * op.n * (2 + (2 if op.w3 else 0) + 4), 0.0
    if kind == "join":
        return T * op.n * (4 + 4 + 4 + (4 if op.in2_slot >= 0 else 0) + (4 if op.add else 0) + (2 if op.out_slot >= 0 else 0)), 0.0
    if kind == "gated_recurrence":
        size = op.n // op.blocks
        return 2 * 2 * op.n * size + T * op.n * (4 + 4 + 2) + B * op.n * 8, 4.0 * T * op.n * size
    if kind in ("layernorm", "norm"):
        return T * op.n * (4 + 4 + 4 + 2), 0.0
    if kind == "cast":
        return T * op.n * 6, 0.0
    if kind == "norm_add":
        return T * op.n * (4 + 4 + 4 + 2 + (2 if op.out2_slot >= 0 else 0)), 0.0
    if kind == "norm_pair":
        return T * op.n * (4 + 2 + (2 if op.out2_slot >= 0 else 0)) + B * op.n * 8, 0.0
    if kind == "reinject":
        return 2 * op.n * op.k + T * (8 * op.n + 2 * 2 * op.k + 8 * op.n), 2.0 * T * op.n * op.k
    if kind == "latent_qkv":
        queries = op.q_rank if op.q_rank else op.heads * (op.head_dim + op.rot_width)       # the queries' latent, or the heads' queries
        row = op.rank + op.rot_width if op.k_off >= 0 else 0
        return 4 * T * (queries + row) + 2 * T * (queries + row), 0.0
    if kind == "head_linear":
        return 2 * op.heads * op.n * op.k + 2 * T * op.heads * (op.k + op.n), 2.0 * T * op.heads * op.n * op.k
    if kind == "latent_attention":
        width = op.rank + op.rot_width
        reach = min(context, op.window) if op.window else context
        keys = B * reach if decode else T
        seen = (B * reach) if decode else sum(min(t + 1, reach) for t in range(T))
        return keys * width * 2 + 2 * T * op.heads * (width + op.rank), 2.0 * seen * op.heads * (width + op.rank)
    if kind == "causal_conv":
        return T * op.n * (4 + 4 + 2), 2.0 * T * op.n * op.taps
    if kind == "selective_scan":
        return T * op.n * (4 + 4 + 2) + 4 * T * (op.rank + 2 * op.k) + 2 * B * op.n * op.k * 4, T * op.n * (6.0 * op.k + 2.0 * op.rank)
    if kind == "delta_rule":
        state = B * op.heads * op.head_dim * dv * 4 * 2
        return state + 4 * T * (op.ld + 2 * op.heads + op.heads * dv) + (4 + 2) * T * op.heads * dv, 6.0 * T * op.heads * op.head_dim * dv
    if kind == "add_rows":
        return T * op.n * (4 + 4 + 2), 0.0
    if kind == "experts":
        pairs = T * op.top * op.experts / (op.experts + op.identity)         # random routers: choices of units with matrices, on average
        used = min(op.experts, pairs)
        return (used * 3 * op.n * op.ff * 2 + T * op.n * (2 + (8 if op.into_stream == 2 else 4)) + pairs * (op.ff * 4 + op.n * 8),
                2.0 * pairs * 3 * op.n * op.ff)
    return 0, 0.0


def run_design(args):
    """Prefill and decode of another design (Sitelorn, Vunelix, Vipovik, Fapenex, Fupapel, Piratar) at layer sizes of real models beside the decoder (llama graph) of
    the same width, feed-forward, heads and layer count (Vipovik: also beside Sitelorn, Fapenex: also beside Vunelix, Fupapel: also
    beside Fapenex, Piratar: also beside Vipovik and Fupapel, the designs closest to them), and every kind
    of launch record of each timed alone against its roofline.  Prints one JSON line of its own kind; the default benchmark is
    untouched."""
    import torch
    from infinicore_infer_b200.config import FapenexConfig, FupapelConfig, MiniCPMConfig, PiratarConfig, SitelornConfig, VipovikConfig, VunelixConfig
    from infinicore_infer_b200.engine import Engine, StepEntry
    from infinicore_infer_b200.parts import model_manifest
    from infinicore_infer_b200.parts.program import OP_NAMES
    from infinicore_infer_b200.weights import DeviceRandomWeights
    from infinicore_infer_b200 import kernels

    peaks, peak_source = load_peaks()
    dev, page = "cuda:0", 16
    T, B, context = args.design_prompt, args.batch, args.design_context
    out = {"design": args.design, "peak_source": peak_source, "peak_hbm_gbs": peaks["hbm_gbs"], "peak_bf16_tflops": peaks["bf16_tflops"],
           "f32_fma_tflops_nominal": round(F32_FMA_TFLOPS, 1), "prompt": T, "decode_batch": B, "decode_context": context,
           "window": args.design_window, "dtype": "bf16", "data": "synthetic: random-init weights, random token ids, synthetic cache", "sizes": {}}
    gen = torch.Generator().manual_seed(0)
    with ClockSampler() as clocks:
        for size in args.design_sizes.split(","):
            width, ff, heads, kv_heads, dim, vocab = DESIGN_SIZES[size]
            block = out["sizes"][size] = {"width": width, "ff": ff, "heads": heads, "kv_heads": kv_heads, "head_dim": dim, "layers": 8}
            beside = {"vipovik": ("sitelorn",), "fapenex": ("vunelix",), "fupapel": ("fapenex",), "piratar": ("vipovik", "fupapel")}.get(args.design, ())
            for which in (args.design,) + beside + ("decoder",):
                if which == "piratar":
                    cfg = PiratarConfig.from_dict(piratar_shape(width, ff, heads, kv_heads, dim, vocab), max_tokens=max(4096, context + page))
                elif which == "fupapel":
                    cfg = FupapelConfig.from_dict(fupapel_shape(width, ff, heads, kv_heads, dim, vocab, args.design_window),
                                                  max_tokens=max(4096, context + page))
                elif which == "fapenex":
                    cfg = FapenexConfig.from_dict(fapenex_shape(width, ff, heads, kv_heads, dim, vocab, args.design_window),
                                                  max_tokens=max(4096, context + page))
                elif which == "vipovik":
                    cfg = VipovikConfig.from_dict(vipovik_shape(width, ff, heads, kv_heads, dim, vocab, args.design_window),
                                                  max_tokens=max(4096, context + page))
                elif which == "vunelix":
                    cfg = VunelixConfig.from_dict(vunelix_shape(width, ff, heads, dim, vocab), max_tokens=max(4096, context + page))
                elif which == "sitelorn":
                    cfg = SitelornConfig.from_dict(sitelorn_shape(width, ff, heads, kv_heads, dim, vocab, args.design_window),
                                                   max_tokens=max(4096, context + page))
                else:
                    cfg = MiniCPMConfig.from_dict(decoder_shape(width, ff, heads, kv_heads, dim, vocab))
                spec = cfg.model_spec()
                weights = DeviceRandomWeights(model_manifest(spec), seed=0, compute_dtype=torch.bfloat16, device=dev, std=0.02, untied=True)
                engine = Engine(spec, weights, dtype=torch.bfloat16, device=dev, cache_tokens=B * (context + page) + T + 4 * page,
                                page_size=page, max_requests=B + 1, max_step_tokens=max(T, 256))
                for view in engine.cache.views:
                    if hasattr(view, "k_pages"):
                        view.k_pages.normal_(0, 0.5); view.v_pages.normal_(0, 0.5)
                    elif hasattr(view, "state") and view.state is not None and view.state.dtype == torch.float32:
                        view.state.normal_(0, 0.1)
                V = spec.vocab_size
                res = block[which] = {}
                # prefill: one prompt of T tokens, the best of three after a warm-up
                ptoks = torch.randint(0, V, (T,), generator=gen).tolist()
                times = []
                for i in range(4):
                    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                    torch.cuda.synchronize()
                    e0.record()
                    engine.step([StepEntry(f"p{i}", ptoks, [T - 1])])
                    e1.record()
                    torch.cuda.synchronize()
                    engine.end(f"p{i}")
                    if i:
                        times.append(e0.elapsed_time(e1))
                res["prefill_ms"] = round(min(times), 3)
                res["prefill_tok_s"] = round(T * 1000.0 / min(times), 1)
                # decode: B requests whose caches hold about `context` positions
                steps, warm = args.steps, max(3, args.warmup)
                start = context - steps - warm - 1
                ids = [f"d{i}" for i in range(B)]
                for r in ids:
                    engine.begin(r); engine.cache.reserve(r, start); engine.cache.commit(r, start)
                entries = [StepEntry(r, [int(t)], [0]) for r, t in zip(ids, torch.randint(0, V, (B,), generator=gen))]
                arg = torch.empty(B, dtype=torch.int32, device=dev)
                for _ in range(warm):
                    kernels.argmax(engine.step(entries), arg)
                torch.cuda.synchronize()
                e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                l0 = engine.kernel_launches
                e0.record()
                for _ in range(steps):
                    kernels.argmax(engine.step(entries), arg)
                e1.record()
                torch.cuda.synchronize()
                ms = e0.elapsed_time(e1) / steps
                res["decode_ms"] = round(ms, 4)
                res["decode_tok_s"] = round(B * 1000.0 / ms, 1)
                res["decode_launches_per_step"] = (engine.kernel_launches - l0) // steps
                engine.check()
                # every kind of record alone, decode then prefill
                prog = engine.program
                if not args.no_kernels:
                    pos = engine.cache.length(ids[0])
                    for r in ids:
                        engine.cache.reserve(r, pos + 1)
                    names, costs = {}, {}
                    for i in range(prog.count):
                        kind = OP_NAMES.get(prog.ops[i].kind)
                        if kind in ("embed",):
                            continue
                        op = prog.ops[i]
                        key = f"{kind}:{op.n}x{op.k}" if kind in ("linear", "gate_up", "residual", "qkv", "head_linear") else \
                            (f"{kind}:{'projected' if op.rank else 'constant'}" if kind == "linear_attention" else kind)
                        # records of one kind that move other amounts (two forms of it in one model) are rows of their own
                        cost, base, n = record_cost(op, T, 1, T, False, page), key, 1
                        while costs.setdefault(key, cost) != cost:
                            n += 1
                            key = f"{base}#{n}"
                        if not (op.wanted_rows and kind != "linear"):
                            names.setdefault(key, []).append(i)
                    kern = res["records"] = {key: {"count": len(idx)} for key, idx in names.items()}
                    engine.begin("kp"); engine.cache.reserve("kp", T)
                    # one phase after the other: a step's metadata lives in one device buffer, which the next upload rewrites
                    for phase, rows, nreq, dec in (("decode", B, B, True), ("prefill", T, 1, False)):
                        ctx_ = engine._upload(entries, [pos] * B, B, B) if dec else engine._upload([StepEntry("kp", ptoks, [T - 1])], [0], 1, T)
                        for key, idx in names.items():
                            op, row = prog.ops[idx[0]], kern[key]
                            us = time_records(engine, ctx_, idx if len(idx) > 1 else idx * 2)
                            nbytes, flops = record_cost(op, rows, nreq, pos + 1 if dec else T, dec, page)
                            row[phase + "_us"] = round(us, 2)
                            mem_frac = nbytes / (us * 1e-6) / 1e9 / peaks["hbm_gbs"]
                            peak_f = F32_FMA_TFLOPS if OP_NAMES.get(op.kind) in ("linear_attention", "selective_scan", "causal_conv", "delta_rule") else peaks["bf16_tflops"]
                            flop_frac = flops / (us * 1e-6) / 1e12 / peak_f
                            row[phase + "_frac"] = round(max(mem_frac, flop_frac), 4)
                            row[phase + "_bound"] = "memory" if mem_frac >= flop_frac else "compute"
                    engine.end("kp")
                for r in ids:
                    engine.end(r)
                del engine, weights
                torch.cuda.empty_cache()
    out["clocks"] = clocks.summary()
    print(json.dumps(out))
    return 0


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--context", type=int, default=4096)
    ap.add_argument("--layers", type=int, default=None, help="run fewer layers than the shape has (both numbers are reported)")
    ap.add_argument("--no-points", action="store_true", help="skip the batch 1 / 64 and context 512 points")
    ap.add_argument("--no-prefill", action="store_true")
    ap.add_argument("--no-context-buckets", action="store_true", help="plan every decode step for the model's longest context")
    ap.add_argument("--no-plain", action="store_true", help="skip the plain (one call per operator) baseline")
    ap.add_argument("--no-kernels", action="store_true", help="skip the per-kernel timings")
    ap.add_argument("--profile", default=None, choices=["decode", "prefill"],
                    help="run a few steps between cudaProfilerStart/Stop (for ncu --profile-from-start off) and exit")
    ap.add_argument("--shape", default="2b", choices=["2b", "1b", "8b"],
                    help="layer sizes: 2b is the headline configuration; the others are for profiles and side measurements")
    ap.add_argument("--design", default=None, choices=["sitelorn", "vunelix", "vipovik", "fapenex", "fupapel", "piratar"],
                    help="instead of the benchmark: prefill and decode of this design at real layer sizes beside the decoder of equal size")
    ap.add_argument("--design-sizes", default="2k,4k", help="comma-separated names of " + ", ".join(sorted(DESIGN_SIZES)))
    ap.add_argument("--design-prompt", type=int, default=2048)
    ap.add_argument("--design-context", type=int, default=2048)
    ap.add_argument("--design-window", type=int, default=1024)
    ap.add_argument("--workload", default=None, choices=sorted(WORKLOADS),
                    help="instead of the decode benchmark: a serving-style workload through the scheduler")
    args = ap.parse_args()

    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable":
                          "InfiniCore-Infer has no Python package to install (xmake C++ project) and its device "
                          "libraries infiniop/infinirt/infiniccl are absent; it cannot be built or run here"}))
        return 0
    if args.gpus != 1:
        print(f"bench.py measures a single-GPU engine: --gpus {args.gpus} is not supported, run with --gpus 1")
        return 2
    if args.warmup < 3:
        args.warmup = 3
    if args.workload:
        return run_workload(args.workload, args.layers)
    if args.design:
        return run_design(args)

    import torch
    from infinicore_infer_b200.config import MiniCPMConfig
    from infinicore_infer_b200.engine import Engine, StepEntry
    from infinicore_infer_b200.jiuge import JiugeForCauslLM
    from infinicore_infer_b200.parts import model_manifest
    from infinicore_infer_b200.tasks import InferTask, KVCache
    from infinicore_infer_b200.weights import DeviceRandomWeights
    from infinicore_infer_b200 import kernels

    peaks, peak_source = load_peaks()
    shape = dict({"2b": SHAPE_2B, "1b": SHAPE_1B, "8b": SHAPE_8B}[args.shape])
    shape_name = {"2b": "MiniCPM-2B shape", "1b": "MiniCPM-1B shape", "8b": "FM9G-8B-class shape"}[args.shape]
    full_layers = shape["num_hidden_layers"]
    if args.layers:
        shape["num_hidden_layers"] = args.layers
    shape["max_position_embeddings"] = max(args.context, 4096)
    cfg = MiniCPMConfig.from_dict(shape)
    spec = cfg.model_spec()
    dev = "cuda:0"
    page = 16
    max_b = 1 if args.no_points else 64
    max_b = max(max_b, args.batch)
    cache_tokens = max(max_b * (args.context + page), 2048 + 4 * page)      # the decode points, or the prompt of 2,048 tokens
    t_load = time.time()
    weights = DeviceRandomWeights(model_manifest(spec), seed=0, compute_dtype=torch.bfloat16, device=dev, std=0.02,
                                  untied=not shape["tie_word_embeddings"])
    engine = Engine(spec, weights, dtype=torch.bfloat16, device=dev, cache_tokens=cache_tokens, page_size=page,
                    max_requests=max_b, max_step_tokens=4096, context_buckets=not args.no_context_buckets)
    engine.config = cfg
    for view in engine.cache.views:          # synthetic cache contents
        view.k_pages.normal_(0, 0.5)
        view.v_pages.normal_(0, 0.5)
    torch.cuda.synchronize()
    t_load = time.time() - t_load
    model = JiugeForCauslLM.from_engine(engine)
    V = spec.vocab_size
    gen = torch.Generator().manual_seed(0)
    kv_bytes_per_token = sum(2 * v.k_pages.shape[1] * v.k_pages.shape[3] * v.k_pages.element_size()
                             for v in engine.cache.views)
    weight_bytes = engine.model.weight_bytes_per_step()

    def fill(n_req, length, prefix):
        """n_req requests whose caches hold ``length`` positions (contents are the synthetic values)."""
        ids = []
        for i in range(n_req):
            rid = f"{prefix}{i}"
            engine.begin(rid)
            engine.cache.reserve(rid, length)
            engine.cache.commit(rid, length)
            ids.append(rid)
        return ids

    def drop(ids):
        for rid in ids:
            engine.end(rid)

    def decode_device(n_req, context, steps, warmup):
        """Device time of ``steps`` decode steps (step function + argmax) with fixed token ids."""
        start = context - (steps + warmup) - 1
        ids = fill(n_req, start, "d")
        toks = torch.randint(0, V, (n_req,), generator=gen).tolist()
        out = torch.empty(n_req, dtype=torch.int32, device=dev)
        entries = [StepEntry(r, [t], [0]) for r, t in zip(ids, toks)]
        for _ in range(warmup):
            kernels.argmax(engine.step(entries), out)
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        l0 = engine.kernel_launches
        e0.record()
        for _ in range(steps):
            kernels.argmax(engine.step(entries), out)
        e1.record()
        torch.cuda.synchronize()
        ms = e0.elapsed_time(e1) / steps
        launches = engine.kernel_launches - l0 + steps
        mean_ctx = start + warmup + (steps + 1) / 2
        drop(ids)
        return ms, launches, mean_ctx

    def decode_e2e(n_req, context, steps, warmup):
        """The same through ``batch_infer_one_round``: host token ids in, sampled ids out, every step."""
        start = context - (steps + warmup) - 1
        tasks = []
        for i in range(n_req):
            t = InferTask(i, [int(torch.randint(0, V, (1,), generator=gen))], context + 8, 0.0, 1, 1.0, [])
            kv = KVCache(model)
            engine.cache.reserve(kv.data(), start)
            engine.cache.commit(kv.data(), start)
            t.bind_kvcache(kv)
            t.pos = start
            tasks.append(t)
        for _ in range(warmup):
            for t, tok in zip(tasks, model.batch_infer_one_round(tasks)):
                t.next(tok)
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        w0 = time.perf_counter()
        e0.record()
        for _ in range(steps):
            for t, tok in zip(tasks, model.batch_infer_one_round(tasks)):
                t.next(tok)
        e1.record()
        torch.cuda.synchronize()
        wall_ms = (time.perf_counter() - w0) * 1000 / steps
        ms = max(e0.elapsed_time(e1) / steps, wall_ms)
        for t in tasks:
            t.kvcache().drop(model)
        return ms

    if args.profile:
        if args.profile == "decode":
            ids = fill(args.batch, args.context - 16, "q")
            entries = [StepEntry(r, [1], [0]) for r in ids]
            out = torch.empty(args.batch, dtype=torch.int32, device=dev)
            for _ in range(3):
                kernels.argmax(engine.step(entries), out)
            torch.cuda.synchronize()
            torch.cuda.profiler.start()
            for _ in range(2):
                kernels.argmax(engine.step(entries), out)
            torch.cuda.synchronize()
            torch.cuda.profiler.stop()
        else:
            ptoks = torch.randint(0, V, (2048,), generator=gen).tolist()
            engine.step([StepEntry("w", ptoks, [2047])]); engine.end("w")
            torch.cuda.synchronize()
            torch.cuda.profiler.start()
            engine.step([StepEntry("w", ptoks, [2047])])
            torch.cuda.synchronize()
            torch.cuda.profiler.stop()
        print(json.dumps({"profiled": args.profile, "layers": cfg.num_hidden_layers}))
        return 0

    result_points = {}
    with ClockSampler() as clocks:
        ms, launches, mean_ctx = decode_device(args.batch, args.context, args.steps, args.warmup)
        e2e_ms = decode_e2e(args.batch, args.context, args.steps, args.warmup)
    clock_summary = clocks.summary()
    value = args.batch * 1000.0 / ms
    step_bytes = weight_bytes + args.batch * mean_ctx * kv_bytes_per_token
    achieved = step_bytes / (ms * 1e-3) / 1e9

    prefill = None
    if not args.no_prefill:
        T = 2048
        ptoks = torch.randint(0, V, (T,), generator=gen).tolist()
        times = []
        for i in range(4):
            rid = f"p{i}"
            torch.cuda.synchronize()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            engine.step([StepEntry(rid, ptoks, [T - 1])])
            e1.record()
            torch.cuda.synchronize()
            engine.end(rid)
            if i >= 1:
                times.append(e0.elapsed_time(e1))
        pms = min(times)
        L, d, nh, dh, di = cfg.num_hidden_layers, cfg.hidden_size, cfg.num_attention_heads, cfg.head_dim, cfg.intermediate_size
        nkv = cfg.num_key_value_heads
        per_tok = 2 * L * (d * (nh + 2 * nkv) * dh + nh * dh * d + 3 * d * di)
        flops = T * per_tok + L * 2 * T * T * dh * nh + 2 * d * V
        prefill = {"value": round(T * 1000.0 / pms, 1), "tokens": T, "ms": round(pms, 3),
                   "frac": round(flops / (pms * 1e-3) / (peaks["bf16_tflops"] * 1e12), 4),
                   "frac_of_sustained": round(flops / (pms * 1e-3) / (peaks["bf16_tflops_sustained"] * 1e12), 4),
                   "tflops": round(flops / (pms * 1e-3) / 1e12, 1), "peak_source": peak_source}

    if not args.no_points:
        psteps, pwarm = min(args.steps, 32), 4
        for name, b, c in (("decode_b1", 1, args.context), ("decode_b64", 64, args.context),
                           ("decode_b1_ctx512", 1, 512), ("decode_b8_ctx512", 8, 512), ("decode_b64_ctx512", 64, 512)):
            pm = sorted(decode_device(b, c, psteps, pwarm)[0] for _ in range(3))[1]       # the median of three runs
            result_points[name] = round(b * 1000.0 / pm, 1)

    # ---- each dominant kernel alone ---------------------------------------------------------------------------
    kernel_block = None
    if not args.no_kernels:
        L, d, nh, nkv, dh, di = (cfg.num_hidden_layers, cfg.hidden_size, cfg.num_attention_heads, cfg.num_key_value_heads,
                                 cfg.head_dim, cfg.intermediate_size)
        nq = (nh + 2 * nkv) * dh
        rec = lambda k: (lambda l: 1 + 7 * l + k)             # a layer's records: norm, qkv, attention, o, norm, gate/up, down
        last = 1 + 7 * L + 1                                   # the output product
        kernel_block = {"peak_hbm_gbs": peaks["hbm_gbs"], "peak_bf16_tflops": peaks["bf16_tflops"], "peak_source": peak_source}

        def mem(name, us, nbytes):
            gbs = nbytes / (us * 1e-6) / 1e9
            kernel_block.update({f"{name}_us": round(us, 2), f"{name}_gbs": round(gbs, 1), f"{name}_frac": round(gbs / peaks["hbm_gbs"], 3)})

        def flop(name, us, flops):
            tf = flops / (us * 1e-6) / 1e12
            kernel_block.update({f"{name}_us": round(us, 2), f"{name}_tflops": round(tf, 1), f"{name}_frac": round(tf / peaks["bf16_tflops"], 3)})

        ids = fill(args.batch, args.context - 2, "k")
        entries = [StepEntry(r, [1], [0]) for r in ids]
        for r in ids:
            engine.cache.reserve(r, args.context - 1)
        dctx = engine._upload(entries, [args.context - 2] * args.batch, args.batch, args.batch)
        mem("decode_qkv", time_records(engine, dctx, rec(1)), nq * d * 2)
        mem("decode_attention", time_records(engine, dctx, rec(2)), args.batch * (args.context - 1) * kv_bytes_per_token / L)
        mem("decode_o", time_records(engine, dctx, rec(3)), d * nh * dh * 2)
        mem("decode_gate_up", time_records(engine, dctx, rec(5)), 2 * di * d * 2)
        mem("decode_down", time_records(engine, dctx, rec(6)), d * di * 2)
        mem("decode_lm_head", time_records(engine, dctx, lambda l: last if l < 3 else None), V * d * 2)
        layer_bytes = (nq * d + d * nh * dh + 3 * di * d) * 2
        layer_us = sum(kernel_block[f"decode_{k}_us"] for k in ("qkv", "o", "gate_up", "down"))
        kernel_block["decode_layer_products_us"] = round(layer_us, 2)
        kernel_block["decode_layer_products_frac"] = round(layer_bytes / (layer_us * 1e-6) / 1e9 / peaks["hbm_gbs"], 3)
        drop(ids)
        T = 2048
        ptoks = torch.randint(0, V, (T,), generator=gen).tolist()
        engine.begin("kp")
        engine.cache.reserve("kp", T)
        pctx = engine._upload([StepEntry("kp", ptoks, [T - 1])], [0], 1, T)
        flop("prefill_qkv", time_records(engine, pctx, rec(1)), 2.0 * T * nq * d)
        flop("prefill_attention", time_records(engine, pctx, rec(2)), 2.0 * T * T * dh * nh)
        flop("prefill_o", time_records(engine, pctx, rec(3)), 2.0 * T * d * nh * dh)
        flop("prefill_gate_up", time_records(engine, pctx, rec(5)), 2.0 * T * 2 * di * d)
        flop("prefill_down", time_records(engine, pctx, rec(6)), 2.0 * T * d * di)
        engine.end("kp")

    # ---- the plain path: one call per operator, library products, plain attention, norm kernels, no graphs ------
    plain = None
    vs_baseline = None
    if not args.no_plain:
        rt = engine.runtime
        saved = (rt.library_products_only, rt.plain_attention, rt.fused_norms, engine.runner.one_by_one, engine.use_graphs)
        rt.library_products_only, rt.plain_attention, rt.fused_norms = True, True, False
        engine.runner.one_by_one, engine.use_graphs = True, False
        plain = {"what": "one call per operator, library products, row attention kernel, norm kernels, no CUDA graphs"}
        for b in (1, 8, 64) if not args.no_points else (args.batch,):
            pm, _, _ = decode_device(b, args.context, 6, 3)
            plain[f"decode_b{b}"] = round(b * 1000.0 / pm, 1)
        if not args.no_prefill:
            T = 2048
            ptoks = torch.randint(0, V, (T,), generator=gen).tolist()
            times = []
            for i in range(3):
                torch.cuda.synchronize()
                e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                e0.record()
                engine.step([StepEntry(f"pp{i}", ptoks, [T - 1])])
                e1.record()
                torch.cuda.synchronize()
                engine.end(f"pp{i}")
                if i >= 1:
                    times.append(e0.elapsed_time(e1))
            plain["prefill_ms"] = round(min(times), 3)
            plain["prefill_tok_s"] = round(T * 1000.0 / min(times), 1)
        (rt.library_products_only, rt.plain_attention, rt.fused_norms, engine.runner.one_by_one, engine.use_graphs) = saved
        base = plain.get(f"decode_b{args.batch}")
        vs_baseline = round(value / base, 3) if base else None

    meta_bytes = 4 * (7 * args.batch + 8 + args.batch * engine.cache.max_blocks * len(engine.cache.groups))
    line = {
        "metric": f"decode tok/s @ batch {args.batch} ({shape_name}, context {args.context})",
        "value": round(value, 1), "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
        "ms_per_step": round(ms, 4), "higher_is_better": True, "scaling": "weak", "vs_baseline": vs_baseline,
        "dtype": "bf16", "data": "synthetic: random-init weights N(0,0.02), uniform random token ids, random cache contents",
        "config": {
            "model": shape_name, "layers": cfg.num_hidden_layers, "layers_of_shape": full_layers,
            "hidden": cfg.hidden_size, "heads": cfg.num_attention_heads, "kv_heads": cfg.num_key_value_heads,
            "head_dim": cfg.head_dim, "intermediate": cfg.intermediate_size, "vocab": cfg.vocab_size,
            "tied_embeddings": bool(cfg.tie_word_embeddings), "global_batch": args.batch, "seq_len": args.context,
            "context_len": args.context, "page_size": page, "parallelism": "single GPU",
            "l2": "inputs larger than L2: 5.4 GB of weights and the cache are re-read every step",
            "weights_gb": round(weight_bytes / 1e9, 3), "kv_bytes_per_token": kv_bytes_per_token,
        },
        "e2e": {"value": round(args.batch * 1000.0 / e2e_ms, 1), "unit": "tokens/s",
                "ms_per_step": round(e2e_ms, 4), "h2d_bytes_per_step": meta_bytes, "d2h_bytes_per_step": 4 * args.batch},
        "gpu_launches": int(launches),
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": peaks["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / peaks["hbm_gbs"], 4), "peak_source": peak_source,
                     "bytes_per_step": int(step_bytes)},
        "clocks": clock_summary,
        "load_s": round(t_load, 1),
    }
    if prefill is not None:
        line["prefill"] = prefill
    if result_points:
        line["points"] = result_points
    if plain is not None:
        line["plain"] = plain
        line["baseline"] = "the engine's own plain path (the reference cannot be built here and publishes no number)"
    if kernel_block is not None:
        line["kernels"] = kernel_block
    print(json.dumps(line))
    return 0


if __name__ == "__main__":
    sys.exit(main())
