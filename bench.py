#!/usr/bin/env python3
"""Benchmark: decode tokens per second of the Qwen3-8B shape on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl reference]
    python bench.py --shape 32b            # the Qwen3-32B shape: batch 1/8/32 to context 8192
    python bench.py --workload serve       # continuous batching, the Qwen3-1.7B shape

Default run: the layer sizes of the Qwen3-8B shape with random weights in
bfloat16, a batch of 8 requests decoding at a context of 4096 tokens.  A "step"
is one decode step (one new token per request).  One JSON line is printed with

- ``value``: decoded tokens per second, timed on the device with CUDA events
  around exactly K steps after W warm-up steps (the step replays the engine's
  CUDA graph; token ids are fed from the host, nothing is read back);
- ``e2e``: the same through the Python entry point (``Engine.step``: scheduler,
  pinned host-to-device copy of the step's inputs, device sampling, read-back of
  the sampled ids each step);
- ``prefill``: one step over a 2,048-token prompt, with its fraction of the
  measured bf16 peak;
- ``roofline``: bytes the decode step must read (every weight once, the cache of
  the live requests) over its time, against the measured copy bandwidth;
- ``points``: decode tokens per second at batch 1 and 64, at batch 8 and 64 with
  64-token pages (the run itself has the reference's block size, 16 tokens), and the
  output tokens per second of the continuous-batching workload below;
- ``clocks``: SM clock and throttle reasons sampled during the timed region.

Between timed steps the inputs (15 GB of weights, gigabytes of cache) are far
larger than the 126 MB L2, so no explicit flush is needed.

``--workload serve``: 64 requests with prompts of 128 to 2048 tokens (uniform, seeded) and
256 output tokens each, all submitted at once to ``Engine.add_request`` and driven by
``Engine.step`` (scheduler, mixed steps of prompt portions beside decode tokens, admission
and page churn) on the Qwen3-1.7B shape: output and total tokens per second, mean time to
the first token, mean time between tokens, preemptions, and how the wall time splits
between the host inside ``Engine.step`` and the GPU.
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

QWEN3_8B = dict(
    architectures=["Qwen3ForCausalLM"], model_type="qwen3", num_hidden_layers=36,
    hidden_size=4096, num_attention_heads=32, num_key_value_heads=8, head_dim=128,
    intermediate_size=12288, vocab_size=151936, rope_theta=1e6, rms_norm_eps=1e-6,
    tie_word_embeddings=False, max_position_embeddings=40960, hidden_act="silu",
    attention_bias=False, use_sliding_window=False)
QWEN3_1P7B = dict(QWEN3_8B, num_hidden_layers=28, hidden_size=2048, num_attention_heads=16,
                  num_key_value_heads=8, intermediate_size=6144, tie_word_embeddings=True)
QWEN3_32B = dict(QWEN3_8B, num_hidden_layers=64, hidden_size=5120, num_attention_heads=64,
                 num_key_value_heads=8, intermediate_size=25600)
# shape -> (config, name, context of the decode points, batches: the second is the headline)
SHAPES = {"8b": (QWEN3_8B, "Qwen3-8B", 4096, (1, 8, 64)),
          "1.7b": (QWEN3_1P7B, "Qwen3-1.7B", 4096, (1, 8, 64)),
          "32b": (QWEN3_32B, "Qwen3-32B", 8192, (1, 8, 32))}
CONTEXT = 4096
PREFILL_TOKENS = 2048
PAGE_SIZE = 16          # the reference's block size, and the configuration's


def load_peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        with open(path) as f:
            p = json.load(f)
        return {"hbm_gbs": float(p["hbm_gbs"]), "bf16_tflops": float(p["bf16_tflops"]),
                "source": "measured"}
    return {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


class ClockSampler:
    """nvidia-smi clocks and throttle reasons, sampled every 100 ms while running."""

    QUERY = ("clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.hw_slowdown,"
             "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
             "clocks_event_reasons.sw_power_cap")

    def __init__(self):
        self.rows, self.proc = [], None

    def start(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", "-i", "0", f"--query-gpu={self.QUERY}",
                 "--format=csv,noheader,nounits", "-lms", "100"],
                stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.rows.append([c.strip() for c in line.split(",")])

    def mark(self):
        return len(self.rows)

    def stop(self):
        if self.proc is not None:
            self.proc.terminate()

    def summary(self, a=0, b=None):
        rows = self.rows[a:b] or self.rows
        sm = [float(r[0]) for r in rows if r and r[0].replace(".", "").isdigit()]
        mx = [float(r[1]) for r in rows if len(r) > 1 and r[1].replace(".", "").isdigit()]
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = [n for i, n in enumerate(names)
                   if any(len(r) > 3 + i and r[3 + i] == "Active" for r in rows)]
        return {"sm_mhz": statistics.median(sm) if sm else None,
                "sm_max_mhz": max(mx) if mx else None, "reasons": reasons,
                "samples": len(rows)}


def reference_arm():
    print(json.dumps({
        "impl": "reference",
        "unavailable": "bwasti/binfer is a Bun/TypeScript program (no setup.py or pyproject.toml: "
                       "pip reports 'not installable'); Bun is not installed and cannot be "
                       "installed offline, and its CMake build pins sm_90"}))
    return 0


def fill_cache(engine, runner, n_req, length, vocab, gen):
    """n_req live requests holding ``length`` tokens each, prefilled through the step function."""
    import torch
    from binfer_b200.engine.runner import StepItem
    rids = []
    for i in range(n_req):
        rid = f"bench{i}"
        runner.add_request(rid)
        toks = torch.randint(0, vocab, (length,), generator=gen).tolist()
        for a in range(0, length, 2048):
            runner.step([StepItem(rid, toks[a:a + 2048], [])])
        rids.append(rid)
    torch.cuda.synchronize()
    return rids


def time_decode(runner, sampler, rids, vocab, steps, warmup, gen, clocks=None):
    """Device time of ``steps`` decode steps (graph replay + greedy sampling)."""
    import torch
    from binfer_b200.csrc import ops
    from binfer_b200.engine.runner import StepItem
    from binfer_b200.sampling import SamplingParams
    B = len(rids)
    params = [SamplingParams(temperature=0.0, seed=0) for _ in rids]
    toks = torch.randint(0, vocab, (steps + warmup, B), generator=gen).tolist()

    def one(i):
        logits = runner.step([StepItem(r, [toks[i][b]], [0]) for b, r in enumerate(rids)])
        return sampler.sample_async(logits, params, [0] * B, [[]] * B)

    for i in range(warmup):
        one(i)
    torch.cuda.synchronize()
    a = clocks.mark() if clocks else 0
    l0 = ops.launches()
    g0 = getattr(runner, "graph_kernel_launches", 0)
    start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    start.record()
    for i in range(warmup, warmup + steps):
        one(i)
    end.record()
    torch.cuda.synchronize()
    b = clocks.mark() if clocks else 0
    ms = start.elapsed_time(end)
    launches = (ops.launches() - l0) + (getattr(runner, "graph_kernel_launches", 0) - g0)
    return ms / steps, launches, (a, b)


def serve_workload(engine, vocab, n_req=64, lo=128, hi=2048, n_out=256, seed=0):
    """64 requests at once through Engine.add_request / Engine.step; the measures of the
    reference's live loop (src/serve.ts:280-550): throughput, time to first token, time
    between tokens."""
    import torch
    from binfer_b200.sampling import SamplingParams
    gen = torch.Generator().manual_seed(seed)
    lens = torch.randint(lo, hi + 1, (n_req,), generator=gen).tolist()
    prompts = [torch.randint(0, vocab, (n,), generator=gen).tolist() for n in lens]
    engine.warm_up()
    engine.time_gpu, engine.gpu_spans, engine.step_ms = True, [], []
    pre0 = engine.scheduler.num_preemptions
    torch.cuda.synchronize()
    t0 = time.perf_counter()
    rids = [engine.add_request(p, SamplingParams(max_tokens=n_out, ignore_eos=True, seed=i))
            for i, p in enumerate(prompts)]
    first, last, seen = {}, {}, {r: 0 for r in rids}
    steps = 0
    while engine.has_work():
        arrived = engine.step()
        now = time.perf_counter() - t0
        steps += 1
        for req in arrived:
            n = len(req.output) - req.unresolved
            if n > seen.get(req.rid, 0):
                first.setdefault(req.rid, now)
                last[req.rid] = now
                seen[req.rid] = n
    torch.cuda.synchronize()
    wall = time.perf_counter() - t0
    engine.time_gpu = False
    gpu_ms = sum(a.elapsed_time(b) for a, b, _ in engine.gpu_spans)
    outs = [engine.requests.pop(r) for r in rids]
    n_out_total = sum(len(r.output) for r in outs)
    itl = [(last[r] - first[r]) / (seen[r] - 1) for r in rids if seen[r] > 1]
    return {
        "requests": n_req, "prompt_tokens": sum(lens), "output_tokens": n_out_total,
        "wall_s": wall, "output_tok_s": n_out_total / wall,
        "total_tok_s": (sum(lens) + n_out_total) / wall,
        "ttft_ms_mean": 1e3 * statistics.mean(first.values()),
        "ttft_ms_max": 1e3 * max(first.values()),
        "itl_ms_mean": 1e3 * statistics.mean(itl),
        "preemptions": engine.scheduler.num_preemptions - pre0, "steps": steps,
        "host_step_s": sum(engine.step_ms) / 1e3, "gpu_busy_s": gpu_ms / 1e3,
        "gpu_idle_frac": max(0.0, 1.0 - gpu_ms / 1e3 / wall),
    }


def serve_point(peaks, layers=None, page_size=PAGE_SIZE):
    """The continuous-batching workload on the Qwen3-1.7B shape, with the bound its decode
    steps have (every weight once and the live cache at the copy bandwidth, batch 64)."""
    import torch
    from binfer_b200 import Engine, Qwen3Config
    raw = dict(QWEN3_1P7B)
    full = raw["num_hidden_layers"]
    if layers:
        raw["num_hidden_layers"] = layers
    cfg = Qwen3Config.from_dict(raw)
    engine = Engine(cfg, "bfloat16", random_seed=1, page_size=page_size, max_seq_len=4096,
                    max_batch_size=64, max_tokens_per_step=2048,
                    num_pages=64 * (4096 // page_size) + 64)
    r = serve_workload(engine, cfg.vocab_size)
    weight_bytes = engine.model.weight_bytes()
    mean_ctx = r["prompt_tokens"] / r["requests"] + 128
    step_s = (weight_bytes + 64 * mean_ctx * cfg.kv_bytes_per_token(2)) / (peaks["hbm_gbs"] * 1e9)
    r["decode_bound_tok_s"] = 64 / step_s
    r["layers"], r["layers_of_full_config"] = cfg.num_hidden_layers, full
    engine.runner.check_errors()
    del engine
    torch.cuda.empty_cache()
    return r


# ------------------------------------------------------------- the hybrid design beside Qwen3
# name -> (width, attention heads, kv heads, head size, feed-forward, memory heads, memory key
# size, memory value size): the attention and feed-forward sizes of the Qwen3 shape of that
# name; the matrix memory's sizes follow the published xLSTM models (keys half, values all of
# the width over its heads)
HYBRID_SIZES = {"1.7b": (2048, 16, 8, 128, 6144, 4, 256, 512),
                "8b": (4096, 32, 8, 128, 12288, 8, 256, 512)}


def hybrid_config(size, layers, window=1024, pool=16):
    width, heads, kv, d, ff, mh, mdk, mdv = HYBRID_SIZES[size]
    attn = {"heads": heads, "kv_heads": kv, "dim": d, "vdim": d, "scale": d ** -0.5,
            "mask": {"size": window, "pool": pool}, "rot": {"base": 1e6, "dims": d}}
    out = []
    for i in range(layers):
        if i % 2 == 0:
            out.append({"type": "mlstm", "mlp": None,
                        "mixer": {"heads": mh, "dim": mdk, "vdim": mdv, "gate_cap": 15.0}})
        else:
            mixer = dict(attn, kv_from=i - 2) if i % 4 == 3 else dict(attn)
            out.append({"type": "attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": ff}})
    return {"architecture": "Gukidra", "vocab": 32000, "width": width, "norm": {"eps": 1e-6},
            "embedding": {"scale": 8.0}, "layers": out}


def side_by_side_config(size, layers, window=1024, keep=4):
    """The side-by-side design at the Qwen3 shape of that name: the attention branch has the
    shape's heads, the retention branch heads of 128 x 256 that together are as wide as the
    model, and the mixture of experts has eight experts of which two run, which with the
    shared expert are as many active inner features as the shape's feed-forward."""
    width, heads, kv, d, ff = HYBRID_SIZES[size][:5]
    rh = width // 256
    left = {"heads": heads, "kv_heads": kv, "dim": d, "vdim": d, "conv": 3, "scale": d ** -0.5,
            "mask": {"size": window, "keep_first": keep},
            "rot": {"base": 1e6, "dims": d // 2,
                    "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}
    right = {"heads": rh, "dim": 128, "vdim": 256, "rot": {"base": 1e6, "dims": 128},
             "decay": [1.0 - 2.0 ** (-5 - 4.0 * i / max(1, rh - 1)) for i in range(rh)]}
    mlp = {"kind": "moe", "router": {"experts": 8, "top": 2}, "expert": {"ff": ff // 4},
           "shared": {"ff": ff // 2}}
    layer = {"type": "parallel", "mlp": mlp,
             "mixer": {"left": left, "right": right, "left_scale": 1.0, "right_scale": 1.0}}
    return {"architecture": "Fikotar", "vocab": 32000, "width": width, "norm": {"eps": 1e-5},
            "logit_scale": 1.0, "layers": [layer] * layers}


def looped_config(size, layers=8):
    """The looped design at the Qwen3 shape of that name, ``layers`` layer runs (at least 4):
    latent attention first and last, between them a gated delta rule layer and a side-by-side
    layer that are walked ``(layers - 2) / 2`` times.  The softmax branch has the shape's
    heads; latent attention has as many heads, of 128 plain and 64 rotated sizes, over a
    latent of 512; the delta rule has value heads of 128 that together are as wide as the
    model and half as many key heads; lightning attention has eight heads of 128; the
    feed-forward is the shape's."""
    width, heads, kv, d, ff = HYBRID_SIZES[size][:5]
    mlp = {"kind": "dense", "ff": ff}
    latent = {"type": "latent_attention", "mlp": mlp,
              "mixer": {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512,
                        "scale": 192 ** -0.5, "rot": {"base": 1e4, "dims": 64}}}
    vh = width // 128
    delta = {"type": "delta", "mlp": mlp,
             "mixer": {"heads": vh, "kv_heads": vh // 2, "dim": 128, "vdim": 128, "conv": 4}}
    left = {"heads": heads, "kv_heads": kv, "dim": d, "vdim": d, "scale": d ** -0.5,
            "softcap": 30.0,
            "rot": {"base": 1e6, "dims": d // 2,
                    "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    right = {"heads": 8, "dim": 128, "vdim": 128,
             "decay": [1.0 - 2.0 ** (-5 - 4.0 * i / 7) for i in range(8)]}
    side = {"type": "parallel", "mlp": mlp,
            "mixer": {"left": left, "right": right, "left_scale": 1.0, "right_scale": 1.0}}
    return {"architecture": "Ketopel", "vocab": 32000, "width": width, "norm": {"eps": 1e-5},
            "embedding": {"scale": 1.0}, "layers": [latent, delta, side, latent],
            "loop": {"start": 1, "stop": 3, "times": max(1, (layers - 2) // 2)}}


def state_space_config(size, layers=8):
    """The design with state space layers at the Qwen3 shape of that name: ``layers`` layers
    that repeat (state space, windowed attention, state space, latent attention).  The state
    space layer is twice as wide inside as the model, in heads of 64 with a state of 128,
    eight groups and four taps (the sizes of the published Mamba-2 hybrids); windowed
    attention has the shape's heads and a window of 1,024; latent attention as many heads, of
    128 plain and 64 rotated sizes, over a latent of 512, its queries through a latent of
    three eighths of the width; the mixture has eight experts and two identity experts in
    five groups of which three are kept, two chosen, which with the shared expert are as many
    active inner features as the shape's feed-forward."""
    width, heads, kv, d, ff = HYBRID_SIZES[size][:5]
    mlp = {"kind": "moe", "expert": {"ff": ff // 4}, "shared": {"ff": ff // 2},
           "router": {"experts": 8, "identity": 2, "top": 2, "scale": 1.5,
                      "groups": {"count": 5, "keep": 3}}}
    inner = 2 * width
    ssm = {"type": "mamba2", "mlp": mlp,
           "mixer": {"heads": inner // 64, "vdim": 64, "state": 128, "groups": 8, "conv": 4,
                     "norm_groups": 8}}
    window = {"type": "attention", "mlp": mlp,
              "mixer": {"heads": heads, "kv_heads": kv, "dim": d, "vdim": d, "scale": d ** -0.5,
                        "mask": {"size": 1024}}}
    latent = {"type": "latent_attention", "mlp": mlp,
              "mixer": {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512,
                        "q_rank": 3 * width // 8, "scale": 192 ** -0.5,
                        "rot": {"base": 1e4, "dims": 64}}}
    pattern = [ssm, window, ssm, latent]
    return {"architecture": "Folivik", "vocab": 32000, "width": width, "norm": {"eps": 1e-5},
            "layers": [pattern[i % 4] for i in range(layers)]}


def differential_config(size, layers=8):
    """The differential attention design at the Qwen3 shape of that name: the shape's query and
    key heads, each of two maps of half the shape's head size (so that a token's keys and
    values take as many bytes as the shape's) over values of its head size; every fourth layer
    reads the keys and values of the layer two before it; the feed-forward is dense with the
    shape's inner features in every other layer, else eight experts of a quarter of them in
    four groups of which two are kept, two chosen."""
    width, heads, kv, d, ff = HYBRID_SIZES[size][:5]
    mixer = {"heads": heads, "kv_heads": kv, "dim": d // 2, "vdim": d, "scale": (d // 2) ** -0.5,
             "diff": 0.5, "q_temp": {"coef": 0.1, "every": 1024}}
    dense = {"kind": "dense", "ff": ff, "limit": 7.0}
    moe = {"kind": "moe", "expert": {"ff": ff // 4},
           "router": {"experts": 8, "top": 2, "groups": {"count": 4, "keep": 2}}}
    return {"architecture": "Pabelix", "vocab": 32000, "width": width, "norm": {"eps": 1e-5},
            "layers": [{"type": "attention", "mlp": moe if i % 2 else dense,
                        "mixer": dict(mixer, kv_from=i - 2) if i % 4 == 3 else mixer}
                       for i in range(layers)]}


def projected_config(size, layers=8):
    """The design whose looped passes project the stream, at the Qwen3 shape of that name, in
    ``layers`` layer runs: three layers (latent attention with a dense feed-forward, windowed
    attention with a mixture, latent attention with a mixture) walked ``(layers - 1) // 3`` times,
    then latent and windowed attention with mixtures in turn for what is left.  Windowed attention
    has the shape's heads and a window of 1,024, latent attention as many heads, of 128 plain and
    64 rotated sizes, over a latent of 512; the dense feed-forward is the shape's, the mixture
    eight experts of which two run, which with the shared expert are as many active inner
    features."""
    width, heads, kv, d, ff = HYBRID_SIZES[size][:5]
    dense = {"kind": "dense", "ff": ff}
    moe = {"kind": "moe", "expert": {"ff": ff // 4, "limit": 7.0},
           "shared": {"ff": ff // 2, "limit": 7.0}, "router": {"experts": 8, "top": 2}}
    window = {"type": "attention", "mlp": moe,
              "mixer": {"heads": heads, "kv_heads": kv, "dim": d, "vdim": d, "scale": d ** -0.5,
                        "mask": {"size": 1024}, "rot": {"base": 1e6, "dims": d}}}
    latent = {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512,
              "scale": 192 ** -0.5,
              "rot": {"base": 1e4, "dims": 64, "scaling": {"factor": 4.0, "original": 4096,
                                                           "fast": 32.0, "slow": 1.0}}}
    looped = [{"type": "latent_attention", "mlp": dense, "mixer": latent}, window,
              {"type": "latent_attention", "mlp": moe, "mixer": latent}]
    times = max(1, (layers - 1) // 3)
    tail = [looped[2], window] * layers
    return {"architecture": "Nazorax", "vocab": 32000, "width": width, "norm": {"eps": 1e-5},
            "layers": looped + tail[:max(0, layers - 3 * times)],
            "loop": {"start": 0, "stop": 3, "times": times}}


def hybrid_compare(args, design="hybrid"):
    """Prefill and decode throughput of the hybrid design (matrix-memory layers alternating
    with pooled-window attention layers), or with ``design`` "side_by_side" of the design
    whose layers run convolved window attention beside retention and a mixture of experts,
    at layer sizes of real models, beside the Qwen3 decoder of the same width, heads,
    feed-forward and layer count: one prompt of 2,048
    tokens in one step, and decode steps at --batch (8) requests with 4,096 tokens of context
    (CUDA graphs), each timed with CUDA events after warm-up; then per-kernel times of both
    (event pairs around every launch, eager).  Random weights, bfloat16."""
    import torch
    from binfer_b200 import Engine, Qwen3Config
    from binfer_b200.config import (FikotarConfig, FolivikConfig, GukidraConfig, KetopelConfig,
                                    NazoraxConfig, PabelixConfig)
    from binfer_b200.engine.runner import StepItem
    from binfer_b200.profiling import Profiler
    layers = args.layers or 8
    B, context, ps = args.batch or 8, 4096, args.page_size
    steps, warmup = min(args.steps, 64), max(args.warmup, 3)
    what = {"hybrid": "hybrid design", "side_by_side": "side-by-side design",
            "looped": "looped design", "state_space": "state space design",
            "differential": "differential attention design",
            "projected": "design with projected passes"}[design]
    # the design with state space layers stands beside the looped design, the closest one
    # (latent attention, a recurrence per head, softmax attention), not beside Qwen3
    # (and the one with projected passes beside that: both have latent and windowed attention
    # and a mixture with a shared expert)
    beside = ("the looped design" if design == "state_space" else
              "the state space design" if design == "projected" else "the Qwen3 decoder")
    record = {"metric": what + " beside " + beside + " at equal layer sizes "
                        "(prefill of 2048 tokens; decode at batch %d, context %d)" % (B, context),
              "dtype": "bf16", "data": "synthetic", "layers": layers, "sizes": {}}
    for size in (args.hybrid_sizes.split(",") if args.hybrid_sizes else sorted(HYBRID_SIZES)):
        width, heads, kv, d, ff = HYBRID_SIZES[size][:5]
        qwen = dict(SHAPES[size][0], num_hidden_layers=layers, vocab_size=32000,
                    tie_word_embeddings=True)
        out = {}
        ours = (GukidraConfig.from_dict(hybrid_config(size, layers)) if design == "hybrid"
                else KetopelConfig.from_dict(looped_config(size, layers)) if design == "looped"
                else FolivikConfig.from_dict(state_space_config(size, layers))
                if design == "state_space"
                else PabelixConfig.from_dict(differential_config(size, layers))
                if design == "differential"
                else NazoraxConfig.from_dict(projected_config(size, layers))
                if design == "projected"
                else FikotarConfig.from_dict(side_by_side_config(size, layers)))
        other = (("looped", KetopelConfig.from_dict(looped_config(size, layers)))
                 if design == "state_space" else
                 ("state_space", FolivikConfig.from_dict(state_space_config(size, layers)))
                 if design == "projected" else ("qwen3", Qwen3Config.from_dict(qwen)))
        for name, cfg in ((design, ours), other):
            engine = Engine(cfg, "bfloat16", random_seed=0, num_pages=(B + 1) * (context // ps) + 64,
                            page_size=ps, max_seq_len=context, max_batch_size=B + 1,
                            max_tokens_per_step=2048, cuda_graphs=True)
            runner = engine.runner
            gen = torch.Generator().manual_seed(0)
            vocab = engine.spec.vocab_size
            toks = torch.randint(0, vocab, (PREFILL_TOKENS,), generator=gen).tolist()

            def prefill():
                runner.add_request("pf")
                runner.step([StepItem("pf", toks, [PREFILL_TOKENS - 1])])
                runner.free_request("pf")

            def timed(fn, n, w):
                for _ in range(w):
                    fn()
                torch.cuda.synchronize()
                a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                a.record()
                for _ in range(n):
                    fn()
                b.record()
                torch.cuda.synchronize()
                return a.elapsed_time(b) / n

            pf_ms = timed(prefill, 5, 3)
            rids = fill_cache(engine, runner, B, context - (steps + warmup) - 8, vocab, gen)
            k = [0]

            def decode():
                k[0] += 1
                runner.step([StepItem(r, [(7 * k[0] + i) % vocab], [0]) for i, r in enumerate(rids)])

            dec_ms = timed(decode, steps, warmup)
            runner.check_errors()
            res = {"prefill_ms": round(pf_ms, 3), "prefill_tok_s": round(PREFILL_TOKENS / pf_ms * 1e3),
                   "decode_ms_per_step": round(dec_ms, 4), "decode_tok_s": round(B / dec_ms * 1e3),
                   "weight_gb": round(engine.model.weight_bytes() / 1e9, 3)}
            # per-kernel shares, eager: the decode step of requests that are freed afterwards
            runner._buckets = None
            kernels = {}
            for what, fn in (("prefill", prefill), ("decode", decode)):
                fn(); fn()
                torch.cuda.synchronize()
                prof = Profiler()
                for _ in range(3):
                    fn()
                prof.stop()
                kernels[what] = {kn: [c // 3, round(ms / 3, 4)] for kn, (c, ms) in
                                 sorted(prof.collect().items(), key=lambda kv: -kv[1][1])}
            res["kernels_calls_ms"] = kernels
            out[name] = res
            for r in rids:
                runner.free_request(r)
            del engine, runner
            torch.cuda.empty_cache()
        record["sizes"][size] = out
    print(json.dumps(record))
    return 0


def profile_steps(args):
    """Per-kernel time of one prefill step and of one decode step, eager (event pairs around
    every launch: short kernels read longer than inside a captured step, so shares, not
    sums, are what to read)."""
    import torch
    from binfer_b200 import Engine, Qwen3Config
    from binfer_b200.engine.runner import StepItem
    from binfer_b200.profiling import Profiler
    base, shape_name, context, batches = SHAPES[args.shape]
    raw = dict(base)
    if args.layers:
        raw["num_hidden_layers"] = args.layers
    cfg = Qwen3Config.from_dict(raw)
    B = args.batch or batches[1]
    ps = args.page_size
    engine = Engine(cfg, "bfloat16", random_seed=0, num_pages=B * (context // ps) + 64 + 256,
                    page_size=ps, max_seq_len=context, max_batch_size=B + 1,
                    max_tokens_per_step=2048, cuda_graphs=False)
    runner = engine.runner
    gen = torch.Generator().manual_seed(0)
    toks = torch.randint(0, cfg.vocab_size, (PREFILL_TOKENS,), generator=gen).tolist()

    def prefill():
        runner.add_request("pf")
        runner.step([StepItem("pf", toks, [PREFILL_TOKENS - 1])])
        runner.free_request("pf")

    rids = fill_cache(engine, runner, B, context - 16, cfg.vocab_size, gen)
    decode_items = [StepItem(r, [7 + i], [0]) for i, r in enumerate(rids)]
    n = 3
    for name, fn in ((f"prefill of {PREFILL_TOKENS} tokens", prefill),
                     (f"decode step, batch {B}, context {context}", lambda: runner.step(decode_items))):
        for _ in range(2):
            fn()
        torch.cuda.synchronize()
        prof = Profiler()
        for _ in range(n):
            fn()
        prof.stop()
        rows = sorted(prof.collect().items(), key=lambda kv: -kv[1][1])
        total = sum(ms for _, (_, ms) in rows)
        print(f"\n{shape_name} shape, {cfg.num_hidden_layers} layers: {name} "
              f"(mean of {n}, {total / n:.2f} ms of kernels)")
        for kernel, (calls, ms) in rows:
            print(f"  {kernel:<30}{calls // n:>6} calls{ms / n:>10.3f} ms{100 * ms / total:>7.1f} %")
    runner.check_errors()
    return 0


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=128)
    ap.add_argument("--warmup", type=int, default=4)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--shape", default="8b", choices=sorted(SHAPES),
                    help="layer sizes: the headline's Qwen3-8B, or the 1.7B / 32B shapes")
    ap.add_argument("--workload", default="decode", choices=["decode", "serve"],
                    help="serve: the continuous-batching workload on the Qwen3-1.7B shape")
    ap.add_argument("--batch", type=int, default=None)
    ap.add_argument("--page-size", type=int, default=PAGE_SIZE)
    ap.add_argument("--layers", type=int, default=None,
                    help="fewer layers than the configuration has (named in the record)")
    ap.add_argument("--no-points", action="store_true", help="skip the other batches, the "
                    "16-token pages, the serve workload and the prefill")
    ap.add_argument("--decode-only", action="store_true",
                    help="only the device-timed decode steps (for profiling): no e2e, no points")
    ap.add_argument("--eager", action="store_true", help="no CUDA graphs (for profiling)")
    ap.add_argument("--profile", action="store_true",
                    help="instead of the bench line: per-kernel CUDA events of a prefill of 2,048 "
                         "tokens and of a decode step at --batch (eager launches; the "
                         "reference's spans: src/profiler/profiler.ts:93-479)")
    ap.add_argument("--hybrid", action="store_true",
                    help="instead of the bench line: prefill and decode throughput of the hybrid "
                         "design (matrix memory + pooled-window attention) beside the Qwen3 "
                         "decoder at equal layer sizes, with per-kernel times")
    ap.add_argument("--side-by-side", action="store_true",
                    help="the same for the design whose layers run convolved window attention "
                         "beside retention, with a mixture of experts")
    ap.add_argument("--looped", action="store_true",
                    help="the same for the design whose layers (latent attention, the gated "
                         "delta rule, whole-norm attention beside lightning attention) are "
                         "partly walked several times")
    ap.add_argument("--state-space", action="store_true",
                    help="the same for the design with state space layers (Mamba-2), windowed "
                         "attention with a logarithmic distance bias and latent attention, with "
                         "a grouped router over experts and identity experts; it stands beside "
                         "the looped design instead of Qwen3")
    ap.add_argument("--differential", action="store_true",
                    help="the same for the design with differential attention, dense clamped "
                         "feed-forwards and a mixture of experts with a sigmoid router")
    ap.add_argument("--projected", action="store_true",
                    help="the same for the design whose looped passes project the stream with the "
                         "embedding output (tanh norms, latent attention with sinks, windowed "
                         "attention with biases, clamped experts); it stands beside the design "
                         "with state space layers instead of Qwen3")
    ap.add_argument("--hybrid-sizes", default="",
                    help="with --hybrid, --side-by-side, --looped, --state-space, --differential "
                         "or --projected: 1.7b, 8b or both (default)")
    args = ap.parse_args()
    if args.impl == "reference":
        return reference_arm()
    if args.gpus != 1:
        print(f"bench.py: this engine runs on one GPU; --gpus {args.gpus} is not supported")
        return 2
    args.warmup = max(args.warmup, 3)
    peaks = load_peaks()
    if args.hybrid:
        return hybrid_compare(args)
    if args.side_by_side:
        return hybrid_compare(args, "side_by_side")
    if args.looped:
        return hybrid_compare(args, "looped")
    if args.state_space:
        return hybrid_compare(args, "state_space")
    if args.differential:
        return hybrid_compare(args, "differential")
    if args.projected:
        return hybrid_compare(args, "projected")
    if args.profile:
        return profile_steps(args)
    if args.workload == "serve":
        r = serve_point(peaks, args.layers, args.page_size)
        print(json.dumps({"metric": "continuous batching, 64 requests x [128, 2048] prompt "
                                    "tokens x 256 output tokens (Qwen3-1.7B shape, bf16, 1 B200)",
                          "value": r["output_tok_s"], "unit": "output tokens/s", "n_gpus": 1,
                          "higher_is_better": True, "dtype": "bf16", "data": "synthetic",
                          "impl": "ours", "serve": r}))
        return 0

    import torch
    from binfer_b200 import Engine, Qwen3Config
    from binfer_b200.csrc import ops
    from binfer_b200.engine import make_runner
    from binfer_b200.engine.runner import StepItem

    base, shape_name, context, batches = SHAPES[args.shape]
    raw = dict(base)
    full_layers = raw["num_hidden_layers"]
    if args.layers:
        raw["num_hidden_layers"] = args.layers
    cfg = Qwen3Config.from_dict(raw)
    steps, warmup = args.steps, args.warmup
    B = args.batch or batches[1]
    page_size = args.page_size
    if args.decode_only:
        args.no_points = True
    max_b = max(B, 1 if args.no_points else max(batches))
    pages = max_b * (context // page_size) + 64
    t0 = time.time()
    engine = Engine(cfg, "bfloat16", random_seed=0, num_pages=pages, page_size=page_size,
                    max_seq_len=context, max_batch_size=max_b, max_tokens_per_step=2048,
                    cuda_graphs=not args.eager)
    runner, sampler = engine.runner, engine.sampler
    vocab = cfg.vocab_size
    gen = torch.Generator().manual_seed(0)
    load_s = time.time() - t0

    weight_bytes = engine.model.weight_bytes() - engine.model.embed.numel() * 2 * (
        0 if cfg.tie_word_embeddings else 1)
    kv_per_token = cfg.kv_bytes_per_token(2)

    clocks = ClockSampler()
    clocks.start()

    def decode_point(batch, n_steps, n_warm, run=None):
        run = run or runner
        start_len = context - (n_steps + n_warm)
        rids = fill_cache(engine, run, batch, start_len, vocab, gen)
        ms, launches, span = time_decode(run, sampler, rids, vocab, n_steps, n_warm, gen, clocks)
        mean_ctx = start_len + n_warm + n_steps / 2
        for r in rids:
            run.free_request(r)
        return ms, launches, span, mean_ctx

    def hbm_frac(batch, ms, mean_ctx):
        return (weight_bytes + batch * mean_ctx * kv_per_token) / (ms / 1e3) / 1e9 / peaks["hbm_gbs"]

    # ---- the headline: batch B at the shape's context
    ms_step, launches, span, mean_ctx = decode_point(B, steps, warmup)
    value = B / (ms_step / 1e3)
    bytes_step = weight_bytes + B * mean_ctx * kv_per_token
    achieved = bytes_step / (ms_step / 1e3) / 1e9
    clk = clocks.summary(*span)
    if clk["samples"] < 3:
        # a short timed region falls between two samples of the clock: time it once more,
        # long enough for a few of them (these steps are not the reported ones)
        extra = max(steps, int(600 / max(ms_step, 0.1)))
        _, _, span2, _ = decode_point(B, min(extra, context // 4), warmup)
        clk = clocks.summary(*span2)
        clk["note"] = "sampled over a longer run of the same steps"

    if args.decode_only:
        clocks.stop()
        print(json.dumps({"decode_only": True, "ms_per_step": ms_step, "value": value,
                          "layers": cfg.num_hidden_layers, "batch": B, "shape": args.shape,
                          "page_size": page_size,
                          "roofline_frac": achieved / peaks["hbm_gbs"], "clocks": clk}))
        return 0

    # ---- end to end through the entry point: scheduler, H2D inputs, D2H ids every step
    # (the clock sampler is stopped first: its nvidia-smi queries contend with the host's
    # CUDA calls, which this measurement, unlike the device-timed one, has in its loop)
    clocks.stop()
    # prompts are prefilled in portions, so the requests start decoding a few steps apart;
    # they are given room enough that none finishes (and the batch does not shrink) while
    # the steps are timed
    slack = 2 * B + 8
    prompts = [torch.randint(0, vocab, (context - (steps + warmup) - slack,),
                             generator=gen).tolist() for _ in range(B)]
    from binfer_b200.sampling import SamplingParams
    for p in prompts:
        engine.add_request(p, SamplingParams(max_tokens=steps + warmup + slack - 1,
                                             ignore_eos=True, seed=0))
    while any(r.remaining > 1 or not r.output for r in engine.scheduler.running) \
            or engine.scheduler.waiting:
        engine.step()                                   # prefill portions
    for _ in range(warmup):
        engine.step()
    torch.cuda.synchronize()
    h0, d0 = runner.h2d_bytes + sampler.h2d_bytes, sampler.d2h_bytes
    t1 = time.perf_counter()
    n_e2e = 0
    for _ in range(steps - 1):
        n_e2e += len(engine.step())
    torch.cuda.synchronize()
    e2e_s = time.perf_counter() - t1
    e2e = {"value": n_e2e / e2e_s, "unit": "tokens/s",
           "h2d_bytes_per_step": (runner.h2d_bytes + sampler.h2d_bytes - h0) // max(steps - 1, 1),
           "d2h_bytes_per_step": (sampler.d2h_bytes - d0) // max(steps - 1, 1)}
    while engine.has_work():
        engine.step()

    points, fracs, prefill, serve = {}, {}, None, None
    if not args.no_points:
        for b in batches:
            if b == B:
                continue
            ms_b, _, _, ctx_b = decode_point(b, steps, warmup)
            points[f"decode_b{b}"] = b / (ms_b / 1e3)
            fracs[f"decode_b{b}"] = round(hbm_frac(b, ms_b, ctx_b), 4)
        # ---- prefill of 2,048 tokens in one step
        toks = torch.randint(0, vocab, (PREFILL_TOKENS,), generator=gen).tolist()
        times = []
        for i in range(5):
            runner.add_request("pf")
            torch.cuda.synchronize()
            s, e = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            s.record()
            runner.step([StepItem("pf", toks, [PREFILL_TOKENS - 1])])
            e.record()
            torch.cuda.synchronize()
            times.append(s.elapsed_time(e))
            runner.free_request("pf")
        pf_ms = statistics.median(times[2:])
        L, H, I = cfg.num_hidden_layers, cfg.hidden_size, cfg.intermediate_size
        Q, KV = cfg.num_attention_heads * cfg.head_dim, cfg.num_key_value_heads * cfg.head_dim
        T = PREFILL_TOKENS
        flops = L * (2 * T * (H * (Q + 2 * KV) + Q * H + 3 * H * I)
                     + 4 * cfg.num_attention_heads * cfg.head_dim * T * (T + 1) / 2) \
            + 2 * H * vocab
        prefill = {"value": T / (pf_ms / 1e3), "tokens": T, "ms": pf_ms,
                   "frac": flops / (pf_ms / 1e3) / (peaks["bf16_tflops"] * 1e12)}
        if args.shape == "8b":
            # ---- the same model over a cache of the other page size (64 tokens, or 16)
            other = 64 if page_size != 64 else 16
            second = make_runner(engine.model, engine.env, page_size=other,
                                 num_pages=max(batches) * (context // other) + 64,
                                 max_requests=max(batches))
            second.enable_decode_graphs(max_batch=max(batches), max_seq_len=context)
            for b in (B, max(batches)):
                ms_b, _, _, ctx_b = decode_point(b, steps, warmup, run=second)
                points[f"decode_b{b}_page{other}"] = b / (ms_b / 1e3)
                fracs[f"decode_b{b}_page{other}"] = round(hbm_frac(b, ms_b, ctx_b), 4)
            second.check_errors()
            del second
    runner.check_errors()
    if not args.no_points and args.shape == "8b":
        del engine, runner
        torch.cuda.empty_cache()
        serve = serve_point(peaks)
        points["serve_1p7b_output_tok_s"] = serve["output_tok_s"]

    out = {
        "metric": f"decode tok/s @ batch {B}, context {context} ({shape_name} shape, bf16, 1 B200)",
        "value": value, "unit": "tokens/s", "n_gpus": 1, "steps": steps, "warmup": warmup,
        "ms_per_step": ms_step, "higher_is_better": True, "scaling": "weak",
        "vs_baseline": None, "dtype": "bf16", "data": "synthetic", "impl": "ours",
        "config": {
            "model": f"{shape_name} shape, random weights", "layers": cfg.num_hidden_layers,
            "layers_of_full_config": full_layers, "hidden": cfg.hidden_size,
            "heads": cfg.num_attention_heads, "kv_heads": cfg.num_key_value_heads,
            "head_dim": cfg.head_dim, "intermediate": cfg.intermediate_size,
            "vocab": cfg.vocab_size, "tied": cfg.tie_word_embeddings, "global_batch": B,
            "seq_len": context, "page_size": page_size, "parallelism": "1 GPU",
            "cuda_graphs": not args.eager, "l2": f"inputs larger than L2 (weights {weight_bytes / 1e9:.0f} GB per step)",
            "clocks_sampled": "during the device-timed steps",
            "peaks": peaks["source"],
        },
        "clocks": clk,
        "e2e": e2e,
        "gpu_launches": launches,
        "roofline": {"bound": "hbm", "achieved": achieved, "peak": peaks["hbm_gbs"],
                     "unit": "GB/s", "frac": achieved / peaks["hbm_gbs"]},
        "points": points,
        "points_hbm_frac": fracs,
    }
    if prefill is not None:
        out["prefill"] = prefill
    if serve is not None:
        out["serve"] = serve
    print(json.dumps(out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
