"""Time one of the engine's kernels alone, at a given size, against its roofline.

    python -m binfer_b200.microbench decode_attention --batch 8 --ctx 4096
    python -m binfer_b200.microbench prefill_attention --tokens 2048
    python -m binfer_b200.microbench diff_prefill --tokens 2048 --head-dim 64 --value-dim 128
    python -m binfer_b200.microbench diff_decode --batch 8 --head-dim 64 --value-dim 128
    python -m binfer_b200.microbench gemm --tokens 8 --features 6144 --k 4096 [--library]
    python -m binfer_b200.microbench add_rmsnorm --tokens 8 --hidden 4096
    python -m binfer_b200.microbench add_tanh_norm --tokens 2048 --hidden 4096
    python -m binfer_b200.microbench experts --tokens 2048 --k 2048 --intermediate 6144
    python -m binfer_b200.microbench out_product --tokens 8 --features 2048 --k 17408
    BINFER_B200_TRACE=1 python -m binfer_b200.microbench step_timeline --batch 8 --ctx 4096 --layers 6

Sizes default to the Qwen3-8B shape.  Each kernel runs on a rotation of input sets
larger than the L2 cache, after warm-up, between CUDA events; the line printed gives
microseconds per launch, the bytes or flops the kernel has to move, and the
fraction of the measured peak (``MEASURED_PEAKS.json`` beside the package, else the
stated fallback).  The reference measures its own peaks the same way at run time
(src/profiler/profiler.ts:553-659).  ``--iters 1 --warmup 0`` gives a run small
enough to put under a profiler.

``step_timeline`` runs whole decode steps of a random-weight model of the given layer sizes
(CUDA graphs, as in serving) with the library built for tracing (``BINFER_B200_TRACE=1``
must be set before the first import: the kernels of the step then record the GPU's global
timer when their first block starts, when its dependency wait returns and when it ends)
and prints the last step's events in order, with the time since the previous one.  Library
products are not instrumented; they show as the gaps around the engine's own kernels.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

from .csrc import ops

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BF16 = torch.bfloat16


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        with open(path) as f:
            p = json.load(f)
        return float(p["hbm_gbs"]), float(p["bf16_tflops"]), "measured"
    return 6650.0, 1590.0, "fallback"


GRAPH = True


def timed(fns, iters, warmup):
    """Microseconds per call of fns[i % len(fns)]() (a rotation of input sets).  The calls
    are captured into one CUDA graph, as the engine's decode step is, so that the host's
    launch cost does not hide the time of a short kernel."""
    for i in range(max(warmup, 1)):
        fns[i % len(fns)]()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    if GRAPH and iters > 1:
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g):
            for i in range(iters):
                fns[i % len(fns)]()
        g.replay()
        torch.cuda.synchronize()
        a.record()
        g.replay()
        b.record()
    else:
        a.record()
        for i in range(iters):
            fns[i % len(fns)]()
        b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) * 1e3 / iters


def report(name, us, nbytes=None, flops=None, **extra):
    hbm, tf, src = peaks()
    out = {"kernel": name, "us": round(us, 2), **extra}
    if nbytes is not None:
        out["GB/s"] = round(nbytes / us / 1e3, 1)
        out["frac_of_hbm_peak"] = round(nbytes / us / 1e3 / hbm, 3)
    if flops is not None:
        out["TFLOP/s"] = round(flops / us / 1e6, 1)
        out["frac_of_bf16_peak"] = round(flops / us / 1e6 / tf, 3)
    out["peaks"] = src
    print(json.dumps(out), flush=True)


def _paged_cache(dev, n_req, ctx, nkv, d, ps, sets, scattered=False):
    """Random caches for n_req requests of ctx tokens.  Pages: the eight (128 / ps) of each
    128-key tile side by side in the pool, the tiles themselves in shuffled order, as the
    page pool hands them out; with ``scattered`` every page anywhere."""
    pages_per = -(-ctx // ps)
    run = max(1, 128 // ps)
    pages_per = -(-pages_per // run) * run
    total = n_req * pages_per + 1
    out = []
    for s in range(sets):
        kc = torch.randn(total, nkv, ps, d, device=dev, dtype=BF16)
        vc = torch.randn(total, nkv, ps, d, device=dev, dtype=BF16)
        if scattered:
            perm = (torch.randperm(total - 1, device=dev) + 1).to(torch.int32)
        else:
            runs = torch.randperm((total - 1) // run, device=dev).to(torch.int32)
            perm = (runs[:, None] * run + 1 + torch.arange(run, device=dev, dtype=torch.int32)
                    ).reshape(-1)
        bt = perm[: n_req * pages_per].view(n_req, pages_per).contiguous()
        out.append((kc, vc, bt))
    return out


def decode_attention(a):
    dev = torch.device("cuda:0")
    B, ctx, nh, nkv, d, ps = a.batch, a.ctx, a.heads, a.kv_heads, a.head_dim, a.page_size
    per_set = 2 * B * ctx * nkv * d * 2
    sets = max(2, int(3e8 // per_set) + 1)
    caches = _paged_cache(dev, B, ctx, nkv, d, ps, sets, a.scattered)
    q = torch.randn(B, nh * d, device=dev, dtype=BF16)
    out = torch.empty_like(q)
    sot = torch.arange(B, dtype=torch.int32, device=dev)
    pos = torch.full((B,), ctx - 1, dtype=torch.int32, device=dev)
    err = ops.error_word(dev)
    fns = [lambda c=c: ops.decode_attention(q, c[0], c[1], None, B, sot, pos, c[2], out, nh, nkv, d,
                                            None, d ** -0.5, ctx, err, variant=a.variant)
           for c in caches]
    us = timed(fns, a.iters, a.warmup)
    report("decode_attention", us, nbytes=per_set, batch=B, ctx=ctx, heads=nh, kv_heads=nkv,
           head_dim=d, page_size=ps)


def prefill_attention(a):
    dev = torch.device("cuda:0")
    T, start, nh, nkv, d, ps = a.tokens, a.start, a.heads, a.kv_heads, a.head_dim, a.page_size
    ctx = start + T
    (kc, vc, bt), = _paged_cache(dev, 1, ctx, nkv, d, ps, 1, a.scattered)
    q = torch.randn(T, nh * d, device=dev, dtype=BF16)
    out = torch.empty_like(q)
    items = torch.tensor([[0, 0, T, start]], dtype=torch.int32, device=dev)
    err = ops.error_word(dev)
    fn = lambda: ops.prefill_attention(q, kc, vc, items, 1, T, bt, out, nh, nkv, d, None,
                                       d ** -0.5, err,
                                       variant=a.variant if a.variant in ("umma2", "umma", "mma_sync")
                                       else "auto", max_ctx=ctx if a.splits < 0 else 0,
                                       splits=max(a.splits, 0))
    us = timed([fn], a.iters, a.warmup)
    flops = 4.0 * nh * d * (T * start + T * (T + 1) / 2)
    report("prefill_attention", us, flops=flops, tokens=T, start=start, heads=nh, kv_heads=nkv,
           head_dim=d)


def _diff_cache(dev, a, n_req, ctx, sets):
    """Caches for differential attention: key rows of both maps side by side, 2 * head_dim."""
    keys = _paged_cache(dev, n_req, ctx, a.kv_heads, 2 * a.head_dim, a.page_size, sets, a.scattered)
    return [(kc, torch.randn(*kc.shape[:3], a.value_dim, device=dev, dtype=BF16), bt)
            for kc, _, bt in keys]


def diff_decode(a):
    dev = torch.device("cuda:0")
    B, ctx, nh, nkv, d, dv = a.batch, a.ctx, a.heads, a.kv_heads, a.head_dim, a.value_dim
    per_set = B * ctx * nkv * (2 * d + dv) * 2
    caches = _diff_cache(dev, a, B, ctx, max(2, int(3e8 // per_set) + 1))
    q = torch.randn(B, nh * 2 * d, device=dev, dtype=BF16)
    gate = torch.randn(B, nh * dv, device=dev, dtype=BF16)
    out = torch.empty_like(gate)
    dc = ops.DiffCombine(0.7, 1e-5, 0.5, gate, 0.1, 1024)
    sot = torch.arange(B, dtype=torch.int32, device=dev)
    pos = torch.full((B,), ctx - 1, dtype=torch.int32, device=dev)
    err = ops.error_word(dev)
    variant = a.variant if a.variant in ("persistent", "mma_sync") else "auto"
    fns = [lambda c=c: ops.diff_attention_decode(q, c[0], c[1], None, B, sot, pos, c[2], out, nh,
                                                 d ** -0.5, dc, ctx, err, variant=variant)
           for c in caches]
    us = timed(fns, a.iters, a.warmup)
    report("diff_decode", us, nbytes=per_set, batch=B, ctx=ctx, heads=nh, kv_heads=nkv,
           map_dim=d, value_dim=dv, page_size=a.page_size, variant=variant)


def diff_prefill(a):
    dev = torch.device("cuda:0")
    T, start, nh, d, dv = a.tokens, a.start, a.heads, a.head_dim, a.value_dim
    (kc, vc, bt), = _diff_cache(dev, a, 1, start + T, 1)
    q = torch.randn(T, nh * 2 * d, device=dev, dtype=BF16)
    gate = torch.randn(T, nh * dv, device=dev, dtype=BF16)
    out = torch.empty_like(gate)
    dc = ops.DiffCombine(0.7, 1e-5, 0.5, gate, 0.1, 1024)
    items = torch.tensor([[0, 0, T, start]], dtype=torch.int32, device=dev)
    err = ops.error_word(dev)
    variant = a.variant if a.variant in ("umma", "mma_sync") else "auto"
    fn = lambda: ops.diff_attention_prefill(q, kc, vc, items, 1, T, bt, out, nh, d ** -0.5, dc,
                                            err, max_ctx=start + T, variant=variant)
    us = timed([fn], a.iters, a.warmup)
    flops = 2.0 * 2 * nh * (d + dv) * (T * start + T * (T + 1) / 2)
    report("diff_prefill", us, flops=flops, tokens=T, start=start, heads=nh, kv_heads=a.kv_heads,
           map_dim=d, value_dim=dv, variant=variant)


def gemm(a):
    dev = torch.device("cuda:0")
    M, N, K = a.tokens, a.features, a.k
    sets = max(2, int(3e8 // (N * K * 2)) + 1)
    ws = [(0.05 * torch.randn(N, K, device=dev)).to(BF16) for _ in range(sets)]
    x = torch.randn(M, K, device=dev).to(BF16)
    out = torch.empty(M, N, device=dev, dtype=BF16)
    err = ops.error_word(dev)
    name = "gemm_bf16_tcgen05"
    if a.library:
        name = "gemm_library"
        fns = [lambda w=w: torch.mm(x, w.t(), out=out) for w in ws]
    elif a.pair:
        name = f"gemm_bf16_pair(bn={a.bn})"
        fns = [lambda w=w: ops.gemm_bf16_pair(x, w, out, err, a.bn) for w in ws]
    elif a.cluster:
        name = f"gemm_bf16_cluster(bn={a.bn},cluster={a.cluster})"
        fns = [lambda w=w: ops.gemm_bf16_cluster(x, w, out, err, a.bn, a.cluster) for w in ws]
    else:
        fns = [lambda w=w: ops.gemm_bf16(x, w, out, err, bn=a.bn) for w in ws]
    us = timed(fns, a.iters, a.warmup)
    report(name, us,
           nbytes=(N * K + M * K + M * N) * 2, flops=2.0 * M * N * K, tokens=M, features=N, k=K)


def swiglu(a):
    """The gate/up projection with the activation in its epilogue (--tokens, --intermediate,
    --k); --library times the library's product followed by the activation kernel."""
    dev = torch.device("cuda:0")
    M, I, K = a.tokens, a.intermediate, a.k
    sets = max(2, int(3e8 // (2 * I * K * 2)) + 1)
    ws = [(0.05 * torch.randn(2 * I, K, device=dev)).to(BF16) for _ in range(sets)]
    x = torch.randn(M, K, device=dev).to(BF16)
    out = torch.empty(M, I, device=dev, dtype=BF16)
    gu = torch.empty(M, 2 * I, device=dev, dtype=BF16)
    err = ops.error_word(dev)
    if a.library:
        name = "library product + silu_mul"

        def two(w):
            torch.mm(x, w.t(), out=gu)
            ops.silu_mul(gu, out)
        fns = [lambda w=w: two(w) for w in ws]
    elif a.pair:
        name = f"gemm_bf16_pair(gated,bn={a.bn})"
        fns = [lambda w=w: ops.gemm_bf16_pair(x, w, out, err, a.bn, gated=True) for w in ws]
    else:
        bn = a.bn or ops.gemm_swiglu_plan(I, K, dev)[0]
        name = f"gemm_bf16_swiglu(bn={bn})"
        fns = [lambda w=w: ops.gemm_bf16_swiglu(x, w, out, err, bn) for w in ws]
    us = timed(fns, a.iters, a.warmup)
    report(name, us, nbytes=(2 * I * K + M * K + M * I) * 2, flops=4.0 * M * I * K, tokens=M,
           intermediate=I, k=K)


def add_rmsnorm(a):
    dev = torch.device("cuda:0")
    T, H = a.tokens, a.hidden
    resid = torch.randn(T, H, device=dev)
    delta = torch.randn(T, H, device=dev).to(BF16)
    w = torch.ones(H, device=dev)
    out = torch.empty(T, H, device=dev, dtype=BF16)
    us = timed([lambda: ops.add_rmsnorm(resid, delta, w, out, 1e-6)], a.iters, a.warmup)
    report("add_rmsnorm", us, nbytes=T * H * (4 + 4 + 2 + 2), tokens=T, hidden=H)


def _stream_sets(a):
    """(stream, pending output) pairs that together exceed the L2 cache."""
    dev, T, H = torch.device("cuda:0"), a.tokens, a.hidden
    sets = max(2, min(64, int(3e8 // (T * H * 6)) + 1))
    return [(torch.randn(T, H, device=dev), torch.randn(T, H, device=dev).to(BF16))
            for _ in range(sets)]


def add_tanh_norm(a):
    """The stream's pending add and bias with the tanh norm (--tokens, --hidden), beside
    ``add_rmsnorm`` on the same rotation of inputs, and the pair that a pass starts from."""
    T, H = a.tokens, a.hidden
    sets = _stream_sets(a)
    w, b = torch.ones(H, device="cuda:0"), torch.zeros(H, device="cuda:0")
    out = torch.empty(T, H, device="cuda:0", dtype=BF16)
    pair = torch.empty(T, 2 * H, device="cuda:0", dtype=BF16)
    table = torch.randn(4096, H, device="cuda:0").to(BF16)
    ids = torch.randint(0, 4096, (T,), device="cuda:0", dtype=torch.int32)
    err = ops.error_word(torch.device("cuda:0"))
    report("add_tanh_norm", timed([lambda x=x, d=d: ops.add_tanh_norm(
        x, d, None, b, 0.5, w, b, out) for x, d in sets], a.iters, a.warmup),
        nbytes=T * H * (4 + 4 + 2 + 2), tokens=T, hidden=H)
    report("add_rmsnorm", timed([lambda x=x, d=d: ops.add_rmsnorm(x, d, w, out, 1e-6)
                                 for x, d in sets], a.iters, a.warmup),
           nbytes=T * H * (4 + 4 + 2 + 2), tokens=T, hidden=H)
    report("stream_pair", timed([lambda x=x, d=d: ops.stream_pair(
        x, d, None, b, table, ids, 1.0, pair, err) for x, d in sets], a.iters, a.warmup),
        nbytes=T * H * (4 + 2 + 2 + 4), tokens=T, hidden=H)


def out_product(a):
    """The output product of few tokens with the stream's add and the tanh norm in its epilogue
    (--tokens, --features, --k), beside the product alone and the norm behind it."""
    dev = torch.device("cuda:0")
    M, N, K = a.tokens, a.features, a.k
    ws = [(0.05 * torch.randn(N, K, device=dev)).to(BF16)
          for _ in range(max(2, int(3e8 // (N * K * 2)) + 1))]
    x, resid = torch.randn(M, K, device=dev).to(BF16), torch.randn(M, N, device=dev)
    nw, nb, err = torch.ones(N, device=dev), torch.zeros(N, device=dev), ops.error_word(dev)
    y, out = torch.empty(M, N, device=dev, dtype=BF16), torch.empty(M, N, device=dev, dtype=BF16)
    plan = ops.gemm_cluster_plan(N, K, dev)

    def two(w):
        ops.gemm_bf16_cluster(x, w, y, err, *plan)
        ops.add_tanh_norm(resid, y, None, nb, 0.5, nw, nb, out)
    for name, fn in (("gemm_bf16_cluster_add_tanh", lambda w: ops.gemm_bf16_cluster_add_tanh(
            x, w, resid, nb, 0.5, nw, nb, err, *plan)),
            ("gemm_bf16_cluster + add_tanh_norm", two),
            ("gemm_bf16_cluster", lambda w: ops.gemm_bf16_cluster(x, w, y, err, *plan))):
        report(name, timed([lambda w=w, fn=fn: fn(w) for w in ws], a.iters, a.warmup),
               nbytes=(N * K + M * K) * 2 + M * N * 10, flops=2.0 * M * N * K, tokens=M, features=N, k=K)


def experts(a):
    """The stacked gate/up product of eight experts of --intermediate / 4 and a shared one of half
    of --intermediate (--tokens, --k) with the clamped activation and the tokens' weights in its
    epilogue, beside the library's product followed by ``moe_act``."""
    dev = torch.device("cuda:0")
    M, K, E, ff, sh = a.tokens, a.k, 8, a.intermediate // 4, a.intermediate // 2
    F = E * ff + sh
    ws = [(0.05 * torch.randn(2 * F, K, device=dev)).to(BF16)
          for _ in range(max(2, int(3e8 // (4 * F * K)) + 1))]
    x, err = torch.randn(M, K, device=dev).to(BF16), ops.error_word(dev)
    rw = torch.rand(M, E, device=dev) * (torch.rand(M, E, device=dev) < 0.25)
    act, gu = (torch.empty(M, n * F, device=dev, dtype=BF16) for n in (1, 2))
    k = dict(activation="clamped", limit=7.0, slope=1.702, up_offset=1.0)
    ea = ops.ExpertAct("clamped", 7.0, 7.0, 1.702, 1.0)
    mix = ops.Mixture(rw, E, ff, False, 7.0)

    def two(w):
        torch.mm(x, w.t(), out=gu)
        ops.moe_act(gu, rw, act, E, ff, shared_gate=False, expert_act=ea)
    cases = [("library product + moe_act", two)]
    plan = ops.gemm_swiglu_plan(F, K, dev) if M <= ops.CLUSTER_MAX_TOKENS else None
    if plan:
        cases.insert(0, ("gemm_bf16_swiglu(mixture)", lambda w: ops.gemm_bf16_swiglu(
            x, w, act, err, plan[0], mixture=mix, **k)))
    if M >= 64:
        cases.insert(0, ("gemm_bf16_pair(mixture)", lambda w: ops.gemm_bf16_pair(
            x, w, act, err, gated=True, mixture=mix, **k)))
    for name, fn in cases:
        report(name, timed([lambda w=w, fn=fn: fn(w) for w in ws], a.iters, a.warmup),
               nbytes=(2 * F * K + M * K + M * F) * 2, flops=4.0 * M * F * K, tokens=M, inner=F, k=K)


FP32_TFLOPS_NOMINAL = 148 * 128 * 2 * 1.965e9 / 1e12      # FMA lanes x 2 x the largest SM clock


def scan(a):
    """A recurrence over --tokens tokens of --batch requests, alone: ``linear`` (a decay per
    token and head, q and k shared by groups of heads: the state space layer's), ``delta``
    (the gated delta rule) or ``retention`` (a fixed decay per head), --heads heads with
    --kv-heads heads of q and k, keys (the state's first size) of --state and values of
    --head-dim.  Arithmetic is counted as the recurrence's own multiply-adds (state update and
    read-out: 5 flops a state element and token, the delta rule 9) against the nominal float
    rate of the FMA pipes; there is no measured peak for it."""
    dev = torch.device("cuda:0")
    B, n, H, G, N, P = a.batch, a.tokens, a.heads, a.kv_heads, a.state, a.head_dim
    T = B * n
    err = ops.error_word(dev)
    q_start = torch.arange(0, T + 1, n, device=dev, dtype=torch.int32)
    slots = torch.arange(B, device=dev, dtype=torch.int32)
    state = torch.zeros(B + 1, H * N * P, device=dev)
    o = torch.empty(T, H * P, device=dev)
    sets = []
    for _ in range(2):
        if a.kind == "linear":
            qk = torch.randn(T, 2, G, N, device=dev) * 0.1
            vf = torch.randn(T, H, P, device=dev)
            dec = torch.rand(T, H, device=dev) * 0.2 + 0.8
            sets.append(lambda qk=qk, vf=vf, dec=dec: ops.linear_scan(
                qk, vf, dec, state, q_start, slots, o, B, H, G, N, P, err, max_q=n))
        elif a.kind == "delta":
            qkv = torch.randn(T, 2 * G * N + H * P, device=dev) * 0.1
            gates = torch.rand(T, 2, H, device=dev) * 0.2 + 0.8
            sets.append(lambda qkv=qkv, gates=gates: ops.delta_scan(
                qkv, gates, state, q_start, slots, o, B, H, G, N, P, err, max_q=n))
        else:
            proj = (torch.randn(T, H * (2 * N + P), device=dev) * 0.1).to(BF16)
            dec = torch.rand(H, device=dev) * 0.2 + 0.8
            pos = torch.arange(n, device=dev, dtype=torch.int32).repeat(B)
            sets.append(lambda proj=proj, dec=dec, pos=pos: ops.retention_scan(
                proj, 0, H * N, 2 * H * N, dec, None, pos, state, q_start, slots, o, B, H, N, P,
                1.0, err, max_q=n))
    us = timed(sets, a.iters, a.warmup)
    flops = (9.0 if a.kind == "delta" else 5.0) * T * H * N * P
    out = {"kernel": a.kind + "_scan", "us": round(us, 2), "tokens": n, "requests": B, "heads": H,
           "qk_heads": G, "keys": N, "values": P, "TFLOP/s": round(flops / us / 1e6, 2),
           "frac_of_nominal_fp32": round(flops / us / 1e6 / FP32_TFLOPS_NOMINAL, 3)}
    print(json.dumps(out), flush=True)
    assert int(err.item()) == 0


def step_timeline(a):
    import ctypes
    from . import Engine
    from .config import Qwen3Config
    from .engine.runner import StepItem
    from .sampling import SamplingParams
    from .csrc import build
    if not build.TRACE:
        raise SystemExit("step_timeline: set BINFER_B200_TRACE=1 in the environment")
    dev = torch.device("cuda:0")
    B, ctx = a.batch, a.ctx
    raw = dict(architectures=["Qwen3ForCausalLM"], model_type="qwen3", num_hidden_layers=a.layers,
               hidden_size=a.hidden, num_attention_heads=a.heads, num_key_value_heads=a.kv_heads,
               head_dim=a.head_dim, intermediate_size=a.intermediate, vocab_size=a.vocab,
               rope_theta=1e6, rms_norm_eps=1e-6, tie_word_embeddings=False,
               max_position_embeddings=max(ctx, 4096), hidden_act="silu", attention_bias=False,
               use_sliding_window=False)
    cfg = Qwen3Config.from_dict(raw)
    ps = a.page_size
    eng = Engine(cfg, "bfloat16", random_seed=0, num_pages=B * (-(-ctx // ps)) + 64, page_size=ps,
                 max_seq_len=ctx, max_batch_size=B, max_tokens_per_step=2048, cuda_graphs=True)
    runner, sampler = eng.runner, eng.sampler
    gen = torch.Generator().manual_seed(0)
    steps = 8
    rids = []
    for i in range(B):
        rid = f"t{i}"
        runner.add_request(rid)
        toks = torch.randint(0, cfg.vocab_size, (ctx - steps - 1,), generator=gen).tolist()
        for s0 in range(0, len(toks), 2048):
            runner.step([StepItem(rid, toks[s0:s0 + 2048], [])])
        rids.append(rid)
    params = [SamplingParams(temperature=0.0, seed=0) for _ in rids]
    torch.cuda.synchronize()
    readers = [getattr(ops.lib(), "bf_trace_read_" + f) for f in
               ("elementwise", "qkv_post", "attention_decode_persistent", "attention_decode",
                "gemm_tcgen05_cluster")]
    times = (ctypes.c_ulonglong * 8192)()
    codes = (ctypes.c_int * 8192)()
    events = []
    for i in range(steps):
        if i == steps - 1:
            torch.cuda.synchronize()
            for rd in readers:
                rd(times, codes)                         # empty the lists: only the last step stays
        logits = runner.step([StepItem(r, [int(torch.randint(0, cfg.vocab_size, (1,), generator=gen))],
                                       [0]) for r in rids])
        sampler.sample_async(logits, params, [0] * B, [[]] * B)
    torch.cuda.synchronize()
    for rd in readers:
        n = rd(times, codes)
        events += [(times[i], codes[i]) for i in range(n)]
    events.sort()
    names = {1: "add_rmsnorm", 2: "silu_mul", 3: "qk_norm_rope", 4: "decode_attention",
             5: "attention_merge", 6: "gemm_cluster"}
    phases = ["first block starts", "wait returns", "ends", "partial sums sent",
              "cluster barrier passed", "products done"]
    t0 = prev = events[0][0]
    print(f"# decode step, batch {B}, context {ctx}, {a.layers} layers; microseconds", flush=True)
    for t, c in events:
        print(f"{(t - t0) / 1e3:10.2f} {(t - prev) / 1e3:8.2f}  {names.get(c // 10, '?'):18s} "
              f"{phases[c % 10]}  [{c}]")
        prev = t
    print(json.dumps({"kernel": "step_timeline", "us": round((events[-1][0] - t0) / 1e3, 2),
                      "events": len(events), "batch": B, "ctx": ctx, "layers": a.layers}))


def main(argv=None):
    ap = argparse.ArgumentParser(prog="python -m binfer_b200.microbench", description=__doc__,
                                 formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("kernel", choices=["decode_attention", "prefill_attention", "gemm",
                                       "swiglu", "add_rmsnorm", "step_timeline", "scan",
                                       "diff_decode", "diff_prefill", "add_tanh_norm",
                                       "out_product", "experts"])
    ap.add_argument("--iters", type=int, default=50)
    ap.add_argument("--warmup", type=int, default=5)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--ctx", type=int, default=4096)
    ap.add_argument("--tokens", type=int, default=8)
    ap.add_argument("--start", type=int, default=0, help="tokens already cached (prefill)")
    ap.add_argument("--heads", type=int, default=32)
    ap.add_argument("--kv-heads", type=int, default=8)
    ap.add_argument("--head-dim", type=int, default=128)
    ap.add_argument("--value-dim", type=int, default=128, help="diff_*: size of a value head "
                                                              "(--head-dim: of one map's key)")
    ap.add_argument("--page-size", type=int, default=16)
    ap.add_argument("--scattered", action="store_true",
                    help="decode_attention: no two pages of a tile side by side in the pool")
    ap.add_argument("--hidden", type=int, default=4096)
    ap.add_argument("--kind", default="linear", choices=["linear", "delta", "retention"],
                    help="scan: which recurrence")
    ap.add_argument("--state", type=int, default=128, help="scan: size of a key (the state's rows)")
    ap.add_argument("--layers", type=int, default=6, help="step_timeline: layers of the model")
    ap.add_argument("--intermediate", type=int, default=12288)
    ap.add_argument("--vocab", type=int, default=151936)
    ap.add_argument("--features", type=int, default=6144)
    ap.add_argument("--k", type=int, default=4096)
    ap.add_argument("--bn", type=int, default=0, help="feature rows per tile (0: chosen)")
    ap.add_argument("--library", action="store_true", help="time cuBLAS on the same product")
    ap.add_argument("--splits", type=int, default=-1,
                    help="prefill attention: shares of the keys per block of 256 queries "
                         "(-1: chosen from the context, 1: none)")
    ap.add_argument("--pair", action="store_true",
                    help="gemm, swiglu: the kernel on pairs of SMs (many token rows)")
    ap.add_argument("--cluster", type=int, default=0,
                    help="gemm: split K over clusters of this many CTAs (needs --bn)")
    ap.add_argument("--no-graph", action="store_true", help="launch from the host, no CUDA graph")
    ap.add_argument("--variant", default="auto", choices=["auto", "persistent", "tma", "cp_async", "umma2", "umma", "mma_sync"],
                    help="decode attention: tma or cp_async tile loads; prefill attention: "
                         "umma (tcgen05) or mma_sync")
    a = ap.parse_args(argv)
    if not torch.cuda.is_available():
        print("microbench needs a CUDA device", file=sys.stderr)
        return 1
    ops.lib()
    global GRAPH
    GRAPH = not a.no_graph
    {"decode_attention": decode_attention, "prefill_attention": prefill_attention,
     "gemm": gemm, "swiglu": swiglu, "add_rmsnorm": add_rmsnorm,
     "step_timeline": step_timeline, "scan": scan, "diff_decode": diff_decode,
     "diff_prefill": diff_prefill, "add_tanh_norm": add_tanh_norm,
     "out_product": out_product, "experts": experts}[a.kernel](a)
    return 0


if __name__ == "__main__":
    sys.exit(main())
