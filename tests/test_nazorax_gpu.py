"""The Nazorax design on the GPU against its plain implementation.

Each kernel alone, each mechanism alone (one-layer models whose weights are made so that the
key in question stands out), then whole models in every replay regime, both precisions, with
page pools so small that every page is used again, the stream after every layer run, the
products with fused epilogues, and generation through the engine's own entry point and
scheduler.
"""
import copy
import dataclasses

import pytest
import torch

import helpers as H
import nazorax_plain as P

pytestmark = pytest.mark.gpu

# largest |difference| / largest |logit|, and rms of the difference / rms of the logits.  The
# float32 bounds are the sharp ones; in bfloat16 every product reads activations rounded to
# eight bits.
TOL = {torch.float32: 6e-5, torch.bfloat16: 0.25}
TOL_RMS = {torch.float32: 1e-5, torch.bfloat16: 6e-2}
F64 = torch.float64
BF16 = torch.bfloat16


def _runner(model_dir, dtype, page_size, num_pages, max_requests=4):
    from binfer_b200.engine import make_env, make_runner, model_from_dir
    env = make_env(dtype)
    model = model_from_dir(model_dir, env)
    return make_runner(model, env, page_size=page_size, num_pages=num_pages,
                       max_requests=max_requests)


def _compare(got, ref, dtype, what, tol_scale=1.0):
    """In bfloat16 a router may decide a close call the other way once its input is rounded:
    up to two in a hundred positions may lie over the bound there (they stay out of the rms
    too); in float32 none."""
    assert got, "the trace produced no logits"
    worst, worst_at, over = 0.0, None, []
    for (rid, pos), row in got.items():
        e = H.rel_err(row, ref[rid][pos])
        if not e <= TOL[dtype] * tol_scale:
            over.append((rid, pos))
        if not e <= worst:
            worst, worst_at = e, (rid, pos)
    allowed = 0 if dtype == torch.float32 else len(got) // 50
    assert len(over) <= allowed, (f"{what}: {len(over)} of {len(got)} positions over the bound, "
                                  f"worst relative error {worst:.3g} at {worst_at}")
    keep = [k for k in got if k not in set(over)]
    g = torch.stack([got[k] for k in keep])
    r = torch.stack([ref[rid][pos] for (rid, pos) in keep])
    assert H.rel_rms(g, r) <= TOL_RMS[dtype] * tol_scale, f"{what}: rms error {H.rel_rms(g, r):.3g}"
    for rid, lg in ref.items():
        assert all((rid, p) in got for p in range(lg.shape[0])), f"{what}: {rid} incomplete"


def _all_regimes(reqs, tail=10):
    return {"whole": H.trace_whole(reqs), "tail": H.trace_decode_tail(reqs, tail),
            "portions": H.trace_portions(reqs), "mixed": H.trace_mixed(reqs)}


def _one_layer(layer, vocab=260, width=48, eps=1e-5):
    return {"architecture": "Nazorax", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": [layer]}


@pytest.fixture
def own_products():
    """The engine's own products for every size that they take."""
    from binfer_b200.parts.linear import set_gemm_policy
    set_gemm_policy("own")
    yield
    set_gemm_policy("auto")


class _Seen:
    """Names of the kernels launched inside ``with``."""

    def __enter__(self):
        from binfer_b200.profiling import Profiler
        self.prof, self.names = Profiler(), set()
        return self

    def __exit__(self, *_):
        from binfer_b200.csrc import ops
        self.prof.stop()
        ops.set_profiler(None)
        self.names = set(self.prof.collect())


# ------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("dtype", [torch.float32, BF16], ids=["f32", "bf16"])
@pytest.mark.parametrize("width", [64, 51, 1, 200, 4096])
def test_tanh_norm_with_pending_adds(cuda_device, dtype, width):
    """Every choice of the two pending adds, the bias and the shift; all rows with the sum written
    back, and picked rows with the stream left alone."""
    from binfer_b200.csrc import ops
    g = torch.Generator().manual_seed(width)
    T, dev = 7, cuda_device
    x = torch.randn(T, width, generator=g)
    d1, d2 = (torch.randn(T, width, generator=g).to(dtype) for _ in range(2))
    bias, w, b = (torch.randn(width, generator=g) for _ in range(3))
    rows = torch.tensor([5, 0, 5, 3], dtype=torch.int32)
    on = lambda t, use: t.to(dev) if use else None               # noqa: E731
    tol = 2e-6 if dtype == torch.float32 else 6e-3
    for use in range(16):
        a1, a2, ab, sh = (bool(use & k) for k in (1, 2, 4, 8))
        total = x.double() + (d1.double() if a1 else 0) + (d2.double() if a2 else 0) + (
            bias.double() if ab else 0)
        want = torch.tanh(0.7 * total) * w.double() + (b.double() if sh else 0)
        resid, out = x.to(dev), torch.empty(T, width, dtype=dtype, device=dev)
        ops.add_tanh_norm(resid, on(d1, a1), on(d2, a2), on(bias, ab), 0.7, w.to(dev), on(b, sh), out)
        assert H.rel_err(resid.cpu(), total) <= 1e-6 and H.rel_err(out.float().cpu(), want) <= tol
        resid, out = x.to(dev), torch.empty(4, width, dtype=dtype, device=dev)
        ops.add_tanh_norm(resid, on(d1, a1), on(d2, a2), on(bias, ab), 0.7, w.to(dev), on(b, sh), out,
                          rows=rows.to(dev), write_back=False)
        assert torch.equal(resid.cpu(), x)
        assert H.rel_err(out.float().cpu(), want[rows.long()]) <= tol


@pytest.mark.parametrize("dtype", [torch.float32, BF16], ids=["f32", "bf16"])
@pytest.mark.parametrize("width", [64, 51, 200])
def test_the_pair_that_a_pass_starts_from(cuda_device, dtype, width):
    from binfer_b200.csrc import ops
    g = torch.Generator().manual_seed(width)
    T, vocab, dev = 6, 30, cuda_device
    x = torch.randn(T, width, generator=g)
    d1, d2 = (torch.randn(T, width, generator=g).to(dtype) for _ in range(2))
    bias = torch.randn(width, generator=g)
    table = torch.randn(vocab, width, generator=g).to(dtype)
    ids = torch.tensor([3, 29, 0, 7, 7, 1], dtype=torch.int32)
    err = torch.zeros(1, dtype=torch.int32, device=dev)
    for a1, a2, ab in ((1, 1, 1), (0, 0, 0), (1, 0, 1), (1, 1, 0)):
        resid = x.to(dev)
        pair = torch.empty(T, 2 * width, dtype=dtype, device=dev)
        ops.stream_pair(resid, d1.to(dev) if a1 else None, d2.to(dev) if a2 else None,
                        bias.to(dev) if ab else None, table.to(dev), ids.to(dev), 1.5, pair, err)
        total = x.double() + a1 * d1.double() + a2 * d2.double() + ab * bias.double()
        want = torch.cat([total, table.double()[ids.long()] * 1.5], dim=1)
        assert torch.equal(resid.cpu(), x)
        assert H.rel_err(pair.float().cpu(), want) <= (1e-6 if dtype == torch.float32 else 5e-3)
    assert int(err.item()) == 0
    # an id outside the table sets the error word and leaves zeros there
    ids[2] = vocab
    ops.stream_pair(x.to(dev), None, None, None, table.to(dev), ids.to(dev), 1.0, pair, err)
    assert int(err.item()) != 0 and float(pair[2, width:].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [torch.float32, BF16], ids=["f32", "bf16"])
def test_biases_of_products_whose_consumers_take_none(cuda_device, dtype):
    from binfer_b200.csrc import ops
    g = torch.Generator().manual_seed(4)
    x, bias = torch.randn(9, 37, generator=g), torch.randn(37, generator=g)
    y = torch.randn(9, 37, generator=g).to(dtype)
    resid, yd = x.to(cuda_device), y.to(cuda_device)
    ops.residual_add(resid, yd, bias.to(cuda_device))
    assert H.rel_err(resid.cpu(), x.double() + y.double() + bias.double()) <= 1e-6
    ops.bias_add(yd, bias.to(cuda_device))
    assert H.rel_err(yd.float().cpu(), y.double() + bias.double()) <= (
        1e-6 if dtype == torch.float32 else 5e-3)


@pytest.mark.parametrize("dtype", [torch.float32, BF16], ids=["f32", "bf16"])
@pytest.mark.parametrize("inner", [64, 13])
def test_activation_with_biases_into_a_column_block(cuda_device, dtype, inner):
    from binfer_b200.csrc import ops
    g = torch.Generator().manual_seed(inner)
    gu = (torch.randn(9, 2 * inner, generator=g) * 2).to(dtype)
    bias = torch.randn(2 * inner, generator=g)
    z = gu.double() + bias.double()
    for act, want in (("silu", P.silu(z[:, :inner]) * z[:, inner:]),
                      ("clamped", z[:, :inner].clamp(max=1.1) * torch.sigmoid(
                          1.702 * z[:, :inner].clamp(max=1.1)) * (z[:, inner:].clamp(-1.1, 1.1) + 1))):
        buf = torch.full((9, inner + 24), 7.0, dtype=dtype, device=cuda_device)
        ops.gated_act_mul(gu.to(cuda_device), buf[:, 16:16 + inner], act, 1.1, 1.702, 1.0,
                          bias=bias.to(cuda_device))
        assert H.rel_err(buf[:, 16:16 + inner].float().cpu(), want) <= (
            3e-6 if dtype == torch.float32 else 8e-3)
        assert bool((buf[:, :16] == 7).all()) and bool((buf[:, 16 + inner:] == 7).all())


def _gated_plain(x, w, bias, kind, route_w=None, E=0, ff=0, shared_gate=False, limit=0.0, sh_limit=0.0):
    z = x.double() @ w.double().T + (bias.double() if bias is not None else 0)
    n = z.shape[1] // 2
    g, u = z[:, :n], z[:, n:]
    if kind == "silu":
        out = P.silu(g) * u
    else:
        lim = torch.full((n,), limit, dtype=F64)
        lim[E * ff:] = sh_limit if E else limit
        g, u = torch.minimum(g, lim), torch.minimum(torch.maximum(u, -lim), lim)
        out = g * torch.sigmoid(P.GATE_SLOPE * g) * (u + P.UP_SHIFT)
    if E:
        wt = torch.ones(x.shape[0], n, dtype=F64)
        wt[:, :E * ff] = route_w[:, :E].double().repeat_interleave(ff, dim=1)
        if shared_gate:
            wt[:, E * ff:] = route_w[:, E:E + 1].double()
        out = out * wt
    return out


@pytest.mark.parametrize("tokens,E,ff,ff_sh,width,shared_gate", [
    (1, 8, 256, 512, 256, False), (8, 6, 328, 200, 512, True), (17, 16, 128, 0, 264, False),
    (64, 5, 512, 96, 256, False), (70, 3, 96, 40, 256, True), (300, 8, 64, 96, 192, False),
    (1100, 4, 160, 72, 256, False)])
@pytest.mark.parametrize("kind", ["silu", "clamped"])
def test_gated_products_with_biases_and_mixtures(cuda_device, tokens, E, ff, ff_sh, width,
                                                 shared_gate, kind):
    """The stacked product with everything in its epilogue, for few token rows and for many, into
    a column block: biases without a mixture, and the mixture's weights, some of them zero, with
    the shared expert's own limit."""
    from binfer_b200.csrc import ops
    dev, inner = cuda_device, E * ff + ff_sh
    g = torch.Generator().manual_seed(tokens + E)
    x = torch.randn(tokens, width, generator=g).to(BF16)
    w = (torch.randn(2 * inner, width, generator=g) * 1.5 / width ** 0.5).to(BF16)
    bias = torch.randn(2 * inner, generator=g)
    rw = torch.rand(tokens, E + (1 if shared_gate else 0), generator=g)
    rw = rw * (torch.rand(rw.shape, generator=g) < 0.4)
    k = dict(activation=kind, limit=1.25, slope=1.702, up_offset=1.0)
    xd, wd, err = x.to(dev), w.to(dev), ops.error_word(dev)
    mix = ops.Mixture(rw.to(dev), E, ff, shared_gate, 0.6)
    cases = [(dict(gate_bias=bias.to(dev)), _gated_plain(x, w, bias, kind, limit=1.25)),
             (dict(mixture=mix), _gated_plain(x, w, None, kind, rw, E, ff, shared_gate, 1.25, 0.6))]
    ran = 0
    for extra, want in cases:
        for pad in (0, 16, 4):                    # (4: no 16-byte rows; the pair kernel's plain stores)
            buf = torch.full((tokens, inner + 2 * pad), 3.0, dtype=BF16, device=dev)
            out = buf[:, pad:pad + inner]
            for form in ("few", "many"):
                if form == "few":
                    plan = ops.gemm_swiglu_plan(inner, width, dev) if tokens <= 64 and inner % 8 == 0 else None
                    if not plan or not ops.gemm_bf16_swiglu(xd, wd, out, err, plan[0], **extra, **k):
                        continue
                elif tokens < 64 or ff % 32 or not ops.gemm_bf16_pair(xd, wd, out, err, gated=True,
                                                                      **extra, **k):
                    continue
                ran += 1
                assert H.rel_err(out.float().cpu(), want) <= 8e-3, (form, pad, sorted(extra))
                assert bool((buf[:, :pad] == 3).all()) and bool((buf[:, pad + inner:] == 3).all())
                out.zero_()
    assert ran >= 2 and int(err.item()) == 0


@pytest.mark.parametrize("tokens", [1, 8, 17, 33, 64])
@pytest.mark.parametrize("N,K", [(256, 512), (200, 1024), (520, 264), (1024, 2048)])
def test_product_with_the_add_and_the_tanh_norm(cuda_device, tokens, N, K):
    """resid (+)= x w^T + bias and the norm of the result, as one kernel; with the stream added to
    or replaced, with and without biases."""
    from binfer_b200.csrc import ops
    dev = cuda_device
    g = torch.Generator().manual_seed(tokens + N)
    x = torch.randn(tokens, K, generator=g).to(BF16)
    wide = (torch.randn(N, K + 8, generator=g) / K ** 0.5).to(BF16)
    w = wide[:, 8:]                                # a column block, as a stacked weight has them
    resid, bias = torch.randn(tokens, N, generator=g), torch.randn(N, generator=g)
    nw, nb = torch.randn(N, generator=g), torch.randn(N, generator=g)
    plan = ops.gemm_cluster_plan(N, K, dev)
    assert plan is not None
    err = ops.error_word(dev)
    for assign, with_bias, with_shift in ((0, 1, 1), (1, 0, 1), (0, 0, 0), (1, 1, 0)):
        r = resid.to(dev)
        y = ops.gemm_bf16_cluster_add_tanh(x.to(dev), wide.to(dev)[:, 8:], r,
                                           bias.to(dev) if with_bias else None, 0.6, nw.to(dev),
                                           nb.to(dev) if with_shift else None, err, *plan,
                                           assign=bool(assign))
        total = x.double() @ w.double().T + with_bias * bias.double() + (
            0 if assign else resid.double())
        assert H.rel_err(r.cpu(), total) <= 1e-5
        want = torch.tanh(0.6 * total) * nw.double() + with_shift * nb.double()
        assert y.dtype == BF16 and H.rel_err(y.float().cpu(), want) <= 6e-3
    assert int(err.item()) == 0


@pytest.mark.parametrize("H_,rank,rot,ps", [(7, 80, 32, 16), (3, 16, 0, 8), (16, 512, 64, 16), (40, 48, 32, 64)])
def test_latent_attention_kernel_with_sinks(cuda_device, H_, rank, rot, ps):
    """The tensor-core kernel and its merge with a logit per head in the denominator: below, among
    and far above the scores; prompts, portions inside tiles, single tokens whose keys are shared
    out."""
    from binfer_b200.csrc import ops
    dev, W = cuda_device, rank + rot
    gen = torch.Generator().manual_seed(H_ + rank)
    scale = 1.7 * W ** -0.5
    sinks = torch.linspace(-20.0, 12.0, H_)
    if H_ > 1:
        sinks[-1] = 90.0                           # takes all of the weight
    for reqs in ([(0, 70), (64, 2), (33, 130), (199, 1), (0, 1)], [(300, 1), (63, 1), (0, 1), (129, 1)],
                 [(515, 1)]):
        pages_of = [(c + n + ps - 1) // ps for c, n in reqs]
        order = torch.randperm(sum(pages_of), generator=gen)
        cache = torch.zeros((sum(pages_of) + 1, 1, ps, W), dtype=BF16)
        tables = torch.full((len(reqs), max(pages_of)), -1, dtype=torch.int32)
        qs, positions, q_start, refs, at = [], [], [0], [], 0
        for b, (c, n) in enumerate(reqs):
            rows = (torch.randn((c + n, W), generator=gen) * 0.8).to(BF16)
            mine = order[at:at + pages_of[b]]
            at += pages_of[b]
            tables[b, :pages_of[b]] = mine.to(torch.int32)
            for j in range(c + n):
                cache[mine[j // ps], 0, j % ps] = rows[j]
            q = (torch.randn((n, H_, W), generator=gen) * 1.5).to(BF16)
            qs.append(q)
            positions += list(range(c, c + n))
            q_start.append(q_start[-1] + n)
            for i in range(n):
                keys = rows[:c + i + 1].double()
                s = torch.cat([q[i].double() @ keys.T * scale, sinks.double()[:, None]], dim=1)
                refs.append(torch.softmax(s, -1)[:, :-1] @ keys[:, :rank])
        q, ref = torch.cat(qs).to(dev), torch.stack(refs)
        out = torch.empty((q.shape[0], H_, rank), dtype=BF16, device=dev)
        err = ops.error_word(dev)
        longest = max(c + n for c, n in reqs)
        for max_ctx in (0, longest, longest + 700):
            out.fill_(float("nan"))
            ops.latent_attention(q, cache.to(dev), torch.tensor(q_start, dtype=torch.int32, device=dev),
                                 torch.tensor(positions, dtype=torch.int32, device=dev),
                                 tables.to(dev), out, len(reqs), max(n for _, n in reqs), H_, rank,
                                 scale, err, max_ctx=max_ctx, sinks=sinks.to(dev))
            assert int(err.item()) == 0
            e = H.rel_err(out.float().cpu(), ref)
            assert e <= 1.2e-2, f"{reqs}, longest context given as {max_ctx}: {e:.3g}"
            if H_ > 1:
                assert float(out[:, -1].float().abs().max()) < 1e-6


# ------------------------------------------------------------------ feed-forwards alone
def _ffn_part(cuda_device, dtype, mlp, width, seed):
    from binfer_b200.config import NazoraxConfig
    from binfer_b200.parts.base import BuildEnv, build_ffn
    from binfer_b200.weights import random_tensors
    from binfer_b200.weights.loader import place
    part = build_ffn(NazoraxConfig._mlp(mlp, "mlp."), width, "f.", BuildEnv(dtype, cuda_device))
    w = random_tensors(part.param_specs(), seed, 0.1, 0.3, dtype)
    by_name = {s.name: s for s in part.param_specs()}
    part.load(lambda s: place(w[s.name], by_name[s.name], dtype, cuda_device))
    return part, {n: t.double() for n, t in w.items()}


@pytest.mark.parametrize("dtype", [torch.float32, BF16], ids=["f32", "bf16"])
@pytest.mark.parametrize("mlp,width", [
    (H._naz_moe(8, 2, 32, 0.8, (48, 0.3)), 64), (H._naz_moe(5, 1, 40, 1.2), 50),
    (H._naz_moe(3, 3, 9, 0.5, (7, 0.9)), 51), (H._naz_moe(1, 1, 16, 0.7, (16, 1.5)), 48),
    (H._naz_moe(16, 4, 128, 1.0, (256, 0.4)), 256), (H._naz_dense(96), 64), (H._naz_dense(13), 51),
    (H._naz_dense(2304), 256)])
def test_feed_forwards_alone(cuda_device, dtype, mlp, width):
    """One and two tokens (the chosen experts alone are read), some tokens (the gated product for
    few rows at the wide sizes), and, in bfloat16, as many as the product on pairs of SMs takes."""
    part, w = _ffn_part(cuda_device, dtype, mlp, width, 5)
    g = torch.Generator().manual_seed(width)
    for T in (1, 2, 37) + ((1030,) if dtype == BF16 else ()):
        h = torch.randn(T, width, generator=g).to(dtype)
        hd = h.double()
        want = P.dense(hd, w, "f.") if mlp["kind"] == "dense" else P.mixture(hd, w, "f.", mlp)
        got = part.forward(h.to(cuda_device), None).float().cpu()
        if mlp["kind"] == "moe" and mlp["router"]["top"] < mlp["router"]["experts"]:
            # a choice between two nearly equal logits may go either way: such tokens aside
            z = torch.sort(hd @ w["f.router"].T, dim=1, descending=True).values
            top = mlp["router"]["top"]
            keep = (z[:, top - 1] - z[:, top]) > 1e-4
            assert int((~keep).sum()) <= max(1, T // 20)
            want, got = want[keep], got[keep]
        assert H.rel_err(got, want) <= (4e-6 if dtype == torch.float32 else 2e-2), T


# ------------------------------------------------------------------ mixers alone, marked keys
def _distinct_tokens(n, vocab, seed):
    return torch.randperm(vocab, generator=torch.Generator().manual_seed(seed))[:n].tolist()


def _mark(w, toks, marked, amp):
    """Two directions of the width are taken out of every embedding; ``e_k`` is put back into the
    embedding of the token at the key's position and ``e_q`` into that of the token at the
    query's.  The layer's norm is nearly the identity (a small alpha, a weight that undoes it),
    and the output head is blind to both."""
    gen = torch.Generator().manual_seed(9)
    width, dt = w["embed"].shape[1], w["embed"].dtype
    e_k = torch.randn(width, generator=gen)
    e_k = e_k / e_k.norm()
    e_q = torch.randn(width, generator=gen)
    e_q = e_q - (e_q @ e_k) * e_k
    e_q = e_q / e_q.norm()
    e_k, e_q = e_k.to(dt), e_q.to(dt)
    for e in (e_k, e_q):
        w["embed"] -= torch.outer(w["embed"] @ e, e)
        w["head"] -= torch.outer(w["head"] @ e, e)
    w["embed"][toks[marked[0]]] += e_k * amp
    w["embed"][toks[marked[1]]] += e_q * amp
    w["l0.norm1.alpha"].fill_(2.0 ** -6)
    w["l0.norm1"].fill_(64.0)
    w["l0.norm1.b"].fill_(0.0)
    return e_k, e_q, gen


def _stand_out_window(raw, toks, marked, amp=3.0, boost=4.0):
    """Windowed attention: the first query head of every group answers ``e_q`` and the group's key
    head answers ``e_k`` with the same vector in the sizes that are not turned."""
    mx = raw["layers"][0]["mixer"]
    H_, G_, dk, rot = mx["heads"], mx["kv_heads"], mx["dim"], mx["rot"]["dims"]

    def tweak(w):
        p = "l0.mix."
        e_k, e_q, gen = _mark(w, toks, marked, amp)
        a = torch.randn(dk, generator=gen).to(w["embed"].dtype)
        a[:rot] = 0.0
        for g in range(G_):
            h0 = g * (H_ // G_)
            w[p + "q"][h0 * dk:(h0 + 1) * dk] += boost * torch.outer(a, e_q)
            w[p + "k"][g * dk:(g + 1) * dk] += boost * torch.outer(a, e_k)
        for e in (e_k, e_q):
            w[p + "v"] -= torch.outer(w[p + "v"] @ e, e)
        w[p + "v"] *= 3.0
        w[p + "o"] *= 4.0
    return tweak


def _stand_out_latent(raw, toks, marked, amp=3.0, boost=30.0):
    """Latent attention: the down projection writes ``e_k`` into the latent's first number; the
    first head's key expansion turns it, and its query ``e_q``, into one fixed vector of the
    sizes that are not turned.  That head's values and the output projection are made large."""
    mx = raw["layers"][0]["mixer"]
    d, dv = mx["dim"], mx["vdim"]

    def tweak(w):
        p = "l0.mix."
        e_k, e_q, gen = _mark(w, toks, marked, amp)
        a = torch.randn(d, generator=gen).to(w["embed"].dtype)
        w[p + "q"] /= 3.0              # (the helper's sharper scores would compete)
        w[p + "dkv"] /= 3.0
        w[p + "dkv"][0] = 0.3 * e_k
        w[p + "dkv.norm"][:] = 1.0
        w[p + "uk"][:d, 0] = a
        w[p + "q"][:d] += boost * torch.outer(a, e_q)
        w[p + "uv"][:dv] *= 6.0
        w[p + "o"] *= 4.0
    return tweak


# pages of 8: the marked key and the query that asks for it
EDGES = {"far": (3, 230), "first_token": (0, 235), "page_border": (8, 27), "page_end": (7, 24),
         "second_token": (0, 1), "neighbour": (100, 101), "itself_before_last": (237, 239)}
WINDOW = 24
# just inside and just outside a window of 24, in a prompt's part and among the tokens decoded
# alone (the last 100), across the cut between them, at a page's first and last place, at the
# sequence's first tokens
WINDOW_EDGES = {"in_prompt": (77, 100), "out_prompt": (76, 100), "in_decoded": (177, 200),
                "out_decoded": (176, 200), "in_page_start": (8, 31), "out_page_end": (7, 31),
                "first_in": (0, 23), "first_out": (0, 24), "second_out": (1, 25),
                "neighbour": (100, 101), "in_across_the_cut": (130, 150), "out_across_the_cut": (126, 150)}
SMALL_MOE = H._naz_moe(3, 2, 12, 1.5, (8, 0.9))


def _moved(raw, w, toks, key, query, ref):
    """How far the query's logits move with another token in the key's place, or, for a key just
    outside the window, with a window one token wider."""
    size = (raw["layers"][0]["mixer"].get("mask") or {}).get("size")
    if size is not None and query - key >= size:
        wider = copy.deepcopy(raw)
        wider["layers"][0]["mixer"]["mask"]["size"] = size + 1
        return H.rel_err(P.forward(wider, w, toks)[query], ref[query])
    other = list(toks)
    other[key] = next(t for t in range(raw["vocab"]) if t not in toks)
    return H.rel_err(P.forward(raw, w, other)[query], ref[query])


def _edge_case(cuda_device, tmp_path, raw, tweak_of, key, query, case):
    toks = _distinct_tokens(240, raw["vocab"], 21)
    d = H.make_nazorax_dir(tmp_path, "A", raw=raw, tweak=tweak_of(raw, toks, (key, query)), tag=case)
    raw, w = H.read_model_dir(d)
    ref = {"a": P.forward(raw, w, toks)}
    moved = _moved(raw, w, toks, key, query, ref["a"])
    assert moved > 100 * TOL[torch.float32], f"{case}: the key moves the logits by {moved:.3g} only"
    for name, steps in _all_regimes({"a": toks}, tail=100).items():
        got = H.run_trace(_runner(d, torch.float32, 8, H.peak_pages(steps, 8)), steps)
        _compare(got, ref, torch.float32, f"{case}/{name}")


@pytest.mark.parametrize("case", sorted(WINDOW_EDGES))
def test_windowed_attention_alone_at_its_edges(cuda_device, tmp_path, case):
    key, query = WINDOW_EDGES[case]
    raw = _one_layer(H._naz_layer("attention", H._naz_attn(4, 2, 16, 24, WINDOW, 8, scale=0.5),
                                  SMALL_MOE), vocab=400)
    _edge_case(cuda_device, tmp_path, raw, _stand_out_window, key, query, case)


@pytest.mark.parametrize("case", sorted(EDGES))
def test_latent_attention_alone_at_its_edges(cuda_device, tmp_path, case):
    key, query = EDGES[case]
    raw = _one_layer(H._naz_layer("latent_attention",
                                  H._naz_latent(3, 12, 8, 20, 28, scale=0.3, yarn=(3.0, 64, 8.0, 1.0)),
                                  H._naz_dense(24)), vocab=400)
    _edge_case(cuda_device, tmp_path, raw, _stand_out_latent, key, query, case)


@pytest.mark.parametrize("which,case", [("window", c) for c in ("in_prompt", "out_prompt", "in_decoded",
                                                                "out_decoded", "first_out", "out_page_end")]
                         + [("latent", c) for c in sorted(EDGES)])
def test_marked_keys_on_the_tensor_cores(cuda_device, tmp_path, which, case):
    """The marked keys again in bfloat16, with sizes that the tiled kernels take; the profiler shows
    that they ran, and the kernel for any sizes on the same rounded numbers is the sharp
    comparison."""
    from binfer_b200.parts import attention_conv_window, attention_latent
    window = which == "window"
    mod = attention_conv_window if window else attention_latent
    key, query = (WINDOW_EDGES if window else EDGES)[case]
    mixer = (H._naz_attn(4, 2, 48, 16, WINDOW, 16, scale=0.4) if window else
             H._naz_latent(4, 32, 16, 48, 64, scale=0.3, yarn=(3.0, 64, 8.0, 1.0)))
    raw = _one_layer(H._naz_layer("attention" if window else "latent_attention", mixer, SMALL_MOE),
                     vocab=400, width=64)
    toks = _distinct_tokens(240, raw["vocab"], 21)
    tweak = (_stand_out_window if window else _stand_out_latent)(raw, toks, (key, query))
    d = H.make_nazorax_dir(tmp_path, "A", BF16, raw=raw, tweak=tweak, tag=which + case)
    raw, w = H.read_model_dir(d)
    ref = P.forward(raw, w, toks)
    moved = _moved(raw, w, toks, key, query, ref)
    assert moved > 0.3, f"{case}: the key moves the logits by {moved:.3g} only"
    outs = []
    for on in (True, False):
        mod.TENSOR_CORES = on
        got = {}
        try:
            with _Seen() as seen:
                for name, steps in _all_regimes({"a": toks}, tail=100).items():
                    got[name] = H.run_trace(_runner(d, BF16, 8, H.peak_pages(steps, 8)), steps)
        finally:
            mod.TENSOR_CORES = True
        for name in got:
            e = H.rel_err(got[name][("a", query)], ref[query])
            assert e <= 0.25 * moved, (f"{case}/{name} (tensor cores {on}): {e:.3g} where the key "
                                       f"moves {moved:.3g}")
        kernel = "pwm_attention" if window else "latent_attention"
        assert (kernel in seen.names) == on and ("paged_attention_generic" in seen.names) != on
        outs.append(got)
    for name in outs[0]:
        worst = max(H.rel_err(outs[0][name][k], outs[1][name][k]) for k in outs[0][name])
        assert worst <= 0.05, f"{case}/{name}: the two kernels differ by {worst:.3g}"


@pytest.mark.parametrize("heads,d,dr,dv,rank", [(1, 6, 2, 10, 6), (2, 40, 24, 8, 200), (5, 8, 40, 30, 12),
                                                (2, 64, 64, 128, 300), (3, 17, 10, 9, 33)])
@pytest.mark.parametrize("dtype", [torch.float32, BF16], ids=["f32", "bf16"])
def test_latent_attention_sizes(cuda_device, tmp_path, heads, d, dr, dv, rank, dtype):
    raw = _one_layer(H._naz_layer("latent_attention",
                                  H._naz_latent(heads, d, dr, dv, rank, yarn=(2.0, 20, 5.0, 1.0)),
                                  H._naz_dense(20)), width=40)
    dd = H.make_nazorax_dir(tmp_path, "B", dtype, raw=raw, tag=f"s{heads}{d}{dr}{rank}")
    raw, w = H.read_model_dir(dd)
    reqs = {"a": H.random_tokens(70, raw["vocab"], 5), "b": H.random_tokens(9, raw["vocab"], 6)}
    ref = {r: P.forward(raw, w, t) for r, t in reqs.items()}
    for name, steps in _all_regimes(reqs, tail=30).items():
        got = H.run_trace(_runner(dd, dtype, 4, H.peak_pages(steps, 4)), steps)
        _compare(got, ref, dtype, f"latent {heads}x{d}+{dr}/{rank}/{name}")


@pytest.mark.parametrize("window", [1, 2, 7, 64, 65, 500])
def test_windows_small_and_large(cuda_device, tmp_path, window):
    """Windows of one token, below, at and above a key tile and wider than the sequence, in
    bfloat16 on the tiled kernel and on the kernel for any sizes."""
    from binfer_b200.parts import attention_conv_window as mod
    raw = _one_layer(H._naz_layer("attention", H._naz_attn(4, 2, 32, 16, window, 32, scale=0.4),
                                  SMALL_MOE), vocab=300, width=64)
    d = H.make_nazorax_dir(tmp_path, "D", BF16, raw=raw, tag=f"w{window}")
    raw, w = H.read_model_dir(d)
    reqs = {"a": H.random_tokens(150, raw["vocab"], 5), "b": H.random_tokens(66, raw["vocab"], 6)}
    ref = {r: P.forward(raw, w, t) for r, t in reqs.items()}
    outs = []
    for on in (True, False):
        mod.TENSOR_CORES = on
        try:
            got = {}
            for name, steps in _all_regimes(reqs, tail=70).items():
                got[name] = H.run_trace(_runner(d, BF16, 8, H.peak_pages(steps, 8)), steps)
                _compare(got[name], ref, BF16, f"window {window}/{name} (tensor cores {on})")
        finally:
            mod.TENSOR_CORES = True
        outs.append(got)
    for name in outs[0]:
        worst = max(H.rel_err(outs[0][name][k], outs[1][name][k]) for k in outs[0][name])
        assert worst <= 0.05, f"window {window}/{name}: the two kernels differ by {worst:.3g}"


# ------------------------------------------------------------------ the new parts in other arrangements
@pytest.mark.parametrize("dtype", [torch.float32, BF16], ids=["f32", "bf16"])
@pytest.mark.parametrize("norm", ["tanh_norm", "layernorm", "rmsnorm"])
@pytest.mark.parametrize("blocks", [("prenorm", "prenorm"), ("parallel", "prenorm"), ("prenorm", "parallel")])
def test_biased_feed_forwards_and_tanh_norms_in_other_arrangements(cuda_device, tmp_path, dtype, norm,
                                                                   blocks, own_products):
    """Layers with one norm a sublayer and layers with one norm for both, in one model, with each
    kind of norm: the biases that ride on the stream's adds, and the tanh norm behind products of
    either arrangement (fused for few tokens in bfloat16)."""
    from binfer_b200.config.specs import NormSpec
    from binfer_b200.config import NazoraxConfig
    from binfer_b200.engine import make_env, make_runner
    from binfer_b200.parts.model import build_model, param_specs_for
    from binfer_b200.weights import random_tensors
    from binfer_b200.weights.loader import TensorSource
    raw = {"architecture": "Nazorax", "vocab": 90, "width": 256, "norm": {"eps": 1e-5},
           "layers": [H._naz_layer("attention", H._naz_attn(4, 2, 32, 32, 12, 16), H._naz_dense(256)),
                      H._naz_layer("attention", H._naz_attn(2, 1, 64, 48, 30, 64), H._naz_dense(320))]}
    spec = NazoraxConfig.from_dict(raw).to_spec()
    ns = NormSpec(kind=norm, eps=1e-5, bias_suffix=".b" if norm != "rmsnorm" else None)
    spec = dataclasses.replace(spec, final_norm=ns, layers=tuple(
        dataclasses.replace(l, block=b, norm=ns) for l, b in zip(spec.layers, blocks)))
    w = random_tensors(param_specs_for(spec), 3, 0.06, 0.2, dtype)
    w["embed"] *= 10.0
    wd = {n: t.double() for n, t in w.items()}

    def apply_norm(x, name):
        if norm == "tanh_norm":
            return P.tanh_norm(x, wd, name)
        if norm == "rmsnorm":
            return P.rms_norm(x, wd[name], 1e-5)
        c = x - x.mean(-1, keepdim=True)
        return P.rms_norm(c, wd[name], 1e-5) + wd[name + ".b"]

    def plain(toks):
        x = wd["embed"][torch.tensor(toks)]
        for i, (layer, block) in enumerate(zip(raw["layers"], blocks)):
            p = f"l{i}."
            h = apply_norm(x, p + "norm1")
            y = P.windowed_attention(h, wd, p + "mix.", layer["mixer"])
            if block == "parallel":
                x = x + y + P.dense(h, wd, p + "mlp.")
            else:
                x = x + y
                x = x + P.dense(apply_norm(x, p + "norm2"), wd, p + "mlp.")
        return apply_norm(x, "final.norm") @ wd["head"].T

    env = make_env(dtype)
    reqs = {"a": H.random_tokens(40, 90, 5), "b": H.random_tokens(13, 90, 6)}
    ref = {r: plain(t) for r, t in reqs.items()}
    for name, steps in _all_regimes(reqs, tail=12).items():
        runner = make_runner(build_model(spec, env, TensorSource.from_dict(w)), env, page_size=8,
                             num_pages=H.peak_pages(steps, 8), max_requests=4)
        with _Seen() as seen:
            got = H.run_trace(runner, steps)
        _compare(got, ref, dtype, f"{norm}/{blocks}/{name}")
        if dtype == BF16 and name == "tail" and norm == "tanh_norm":
            assert "gemm_bf16_cluster_add_tanh" in seen.names


# ----------------------------------------------------------------------- whole models
LENGTHS = {"A": [5, 17, 33, 70, 121], "B": [1, 9, 40, 70, 101], "C": [3, 30, 64, 47, 2],
           "D": [2, 45, 150, 210, 90]}


def _requests(which, extra=()):
    vocab = H.NAZ[which]["raw"]["vocab"]
    lens = list(LENGTHS[which]) + list(extra)
    return {f"r{i}": H.random_tokens(n, vocab, 100 * i + n) for i, n in enumerate(lens)}


@pytest.fixture(scope="module")
def plain_logits(tmp_path_factory):
    cache = {}

    def get(which, dtype, reqs):
        d = H.make_nazorax_dir(tmp_path_factory.getbasetemp(), which, dtype)
        raw, w = H.read_model_dir(d)
        out = cache.setdefault((which, dtype), {})
        for rid, toks in reqs.items():
            k = (rid, tuple(toks))
            if k not in out:
                out[k] = P.forward(raw, w, toks)
        return d, {rid: out[(rid, tuple(toks))] for rid, toks in reqs.items()}

    return get


@pytest.mark.parametrize("which,dtype", [("A", torch.float32), ("B", torch.float32),
                                         ("C", torch.float32), ("D", torch.float32), ("A", BF16),
                                         ("B", BF16), ("C", BF16), ("D", BF16)],
                         ids=["A-f32", "B-f32", "C-f32", "D-f32", "A-bf16", "B-bf16", "C-bf16", "D-bf16"])
@pytest.mark.parametrize("regime", ["whole", "tail", "portions", "mixed"])
def test_replay(cuda_device, plain_logits, which, dtype, regime):
    """Seven requests, at most four at a time, through page pools of exactly the peak need."""
    reqs = _requests(which, (55, 61) if regime == "mixed" else ())
    model_dir, ref = plain_logits(which, dtype, reqs)
    steps = _all_regimes(reqs)[regime]
    ps = H.NAZ[which]["page_size"]
    runner = _runner(model_dir, dtype, ps, H.peak_pages(steps, ps))
    got = H.run_trace(runner, steps)
    assert not runner.cache.requests and all(g.pool.num_held == 0 for g in runner.cache.groups)
    _compare(got, ref, dtype, f"{which}/{regime}")


@pytest.mark.parametrize("regime", ["whole", "tail", "mixed"])
def test_replay_on_the_fused_products(cuda_device, plain_logits, regime, own_products):
    """The engine's own products wherever they take the sizes: the stream's add and the tanh norm
    in the output product's epilogue, the pass projection with the norm behind it, the experts'
    activation and weighting in the gated product (also the one for many rows)."""
    from binfer_b200.parts import mlp, moe
    reqs = _requests("D", (300,) if regime == "whole" else ())
    model_dir, ref = plain_logits("D", BF16, reqs)
    steps = _all_regimes(reqs)[regime]
    fill = mlp.FUSE_SWIGLU_FILL
    mlp.FUSE_SWIGLU_FILL = moe.FUSE_SWIGLU_FILL = 0.0
    try:
        runner = _runner(model_dir, BF16, 16, H.peak_pages(steps, 16))
        with _Seen() as seen:
            got = H.run_trace(runner, steps)
    finally:
        mlp.FUSE_SWIGLU_FILL = moe.FUSE_SWIGLU_FILL = fill
    _compare(got, ref, BF16, f"fused/{regime}")
    assert {"gemm_bf16_cluster_add_tanh"} <= seen.names
    if regime == "whole":
        assert "gemm_bf16_pair" in seen.names


@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
def test_the_stream_after_every_layer_run(cuda_device, plain_logits, which):
    from binfer_b200.engine.runner import StepItem
    toks = H.random_tokens(19, H.NAZ[which]["raw"]["vocab"], 77)
    model_dir, _ = plain_logits(which, torch.float32, {})
    raw, w = H.read_model_dir(model_dir)
    want = []
    P.forward(raw, w, toks, want)
    runner = _runner(model_dir, torch.float32, 8, 4)
    runner.add_request("a")
    items = [StepItem("a", toks, [len(toks) - 1])]
    runner.reserve(items)
    runner.cache.zero_fresh_state(runner.cache.get("a"))
    ctx = runner.build_context(items)
    ctx.scratch["layer_outputs"] = []
    runner.model.forward(ctx, runner.views)
    got = ctx.scratch["layer_outputs"]
    assert len(got) == len(want) == len(runner.model.spec.schedule)
    for i, (g, r) in enumerate(zip(got, want)):
        assert H.rel_err(g.cpu(), r) <= 2e-5, f"{which}: after layer run {i}"


@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
def test_regimes_agree_bitwise_in_float32(cuda_device, plain_logits, which):
    """Every sum's order depends on positions and sizes alone: cutting and batching change
    no bit."""
    reqs = _requests(which)
    model_dir, _ = plain_logits(which, torch.float32, reqs)
    ps = H.NAZ[which]["page_size"]
    outs = []
    for steps in _all_regimes(reqs).values():
        outs.append(H.run_trace(_runner(model_dir, torch.float32, ps, H.peak_pages(steps, ps)),
                                steps))
    for other in outs[1:]:
        for key, row in outs[0].items():
            assert torch.equal(row, other[key]), f"{which}: logits at {key} depend on the cut"


def test_requests_alone_and_in_a_batch(cuda_device, plain_logits):
    """Unequal requests in one batch give what each gives alone, bit for bit in float32."""
    reqs = _requests("B")
    model_dir, _ = plain_logits("B", torch.float32, reqs)
    together = H.run_trace(_runner(model_dir, torch.float32, 4, 200, 8),
                           [{"step": 0, "end": list(reqs), "entries": [
                               {"id": r, "tokens": t, "want": list(range(len(t)))} for r, t in reqs.items()]}])
    for rid, toks in reqs.items():
        alone = H.run_trace(_runner(model_dir, torch.float32, 4, 200), H.trace_whole({rid: toks}))
        for key, row in alone.items():
            assert torch.equal(row, together[key]), key


@pytest.mark.parametrize("dtype", [torch.float32, BF16], ids=["f32", "bf16"])
def test_long_decoding(cuda_device, plain_logits, dtype):
    """A short prompt, then 300 tokens one by one: the windows pass over decoded tokens and give
    their pages back."""
    reqs = {"long": H.random_tokens(304, H.NAZ["B"]["raw"]["vocab"], 7)}
    model_dir, ref = plain_logits("B", dtype, reqs)
    steps = H.trace_decode_tail(reqs, tail=300)
    _compare(H.run_trace(_runner(model_dir, dtype, 4, 76), steps), ref, dtype, "long decoding")


@pytest.mark.parametrize("which,dtype", [("A", torch.float32), ("D", BF16)], ids=["A-f32", "D-bf16"])
def test_decoding_from_captured_steps(cuda_device, plain_logits, which, dtype):
    """Steps of single tokens replayed from CUDA graphs give what eager steps give."""
    reqs = _requests(which, (55, 61))
    model_dir, ref = plain_logits(which, dtype, reqs)
    steps = H.trace_mixed(reqs, tail=20)
    ps = H.NAZ[which]["page_size"]
    runner = _runner(model_dir, dtype, ps, H.peak_pages(steps, ps))
    runner.enable_decode_graphs(max_batch=4, max_seq_len=256)
    got = H.run_trace(runner, steps)
    assert getattr(runner, "graph_replays", 0) > 0
    _compare(got, ref, dtype, "captured decode steps")


# ------------------------------------------------------------------------- generation
@pytest.mark.parametrize("graphs,step_tokens", [(True, 2048), (False, 7)], ids=["graphs", "portions"])
def test_greedy_generation_through_the_engine(cuda_device, tmp_path, graphs, step_tokens):
    """Prompts of 5/17/33/2 tokens through ``Engine.generate``: the scheduler's admission, portions
    of at most seven tokens beside decoding (second case), captured decode steps (first case);
    every token is the plain implementation's choice."""
    from binfer_b200 import Engine
    d = H.make_nazorax_dir(tmp_path, "A")
    raw, w = H.read_model_dir(d)
    prompts = [H.random_tokens(n, raw["vocab"], n) for n in (5, 17, 33, 2)]
    eng = Engine(d, "float32", num_pages=40, page_size=16, max_seq_len=128, max_batch_size=3,
                 max_tokens_per_step=step_tokens, cuda_graphs=graphs)
    got = eng.generate(prompts, max_tokens=12, ignore_eos=True)
    for p, out in zip(prompts, got):
        assert len(out) == 12
        logits = P.forward(raw, w, list(p) + list(out))
        for n, tok in enumerate(out):
            row = logits[len(p) - 1 + n]
            assert float(row[tok]) >= float(row.max()) - 1e-4 * float(row.abs().max()), (
                f"token {n} after a prompt of {len(p)}: {tok}, plain {int(row.argmax())}")
    st = eng.stats()
    assert st["pages_free"] == st["pages_total"]
    if graphs:
        assert getattr(eng.runner, "graph_replays", 0) > 0


def test_command_line_generates_from_a_folder(cuda_device, tmp_path, capsys):
    from binfer_b200.cli import main
    d = H.make_nazorax_dir(tmp_path, "C")
    raw, w = H.read_model_dir(d)
    prompt = H.random_tokens(9, raw["vocab"], 3)
    ids = ",".join(map(str, prompt))
    common = [d, "--prompt-ids", ids, "--dtype", "fp32", "--ignore-eos", "-q", "--kv-pages", "32"]
    assert main(common + ["--max-tokens", "5"]) == 0
    out = [int(t) for t in capsys.readouterr().out.split()]
    assert len(out) == 5
    logits = P.forward(raw, w, list(prompt) + out)
    for n, tok in enumerate(out):
        row = logits[len(prompt) - 1 + n]
        assert float(row[tok]) >= float(row.max()) - 1e-4 * float(row.abs().max())
    sampled = []
    for _ in range(2):
        assert main(common + ["--max-tokens", "8", "--temperature", "0.9", "--seed", "5"]) == 0
        sampled.append(capsys.readouterr().out.split())
    assert sampled[0] == sampled[1] and len(sampled[0]) == 8


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_tool(cuda_device, tmp_path, dtype):
    """``bin/trace_run`` as a user runs it: six requests, four at a time, through a page pool sized
    by ``--max-tokens``."""
    import test_trace_run_gpu as TR
    dt = getattr(torch, dtype)
    d = H.make_nazorax_dir(tmp_path, "B", dt)
    raw, w = H.read_model_dir(d)
    reqs = {f"r{i}": H.random_tokens(n, raw["vocab"], 31 * i + n)
            for i, n in enumerate([70, 33, 90, 12, 64, 41])}
    steps = H.trace_mixed(reqs)
    live, peak = {}, 0
    for st in steps:
        for e in st["entries"]:
            live[e["id"]] = live.get(e["id"], 0) + len(e["tokens"])
        peak = max(peak, sum(-(-n // 64) * 64 for n in live.values()))
        for rid in st["end"]:
            live.pop(rid)
    out_dir = str(tmp_path / "out")
    TR._replay(d, dtype, steps, out_dir, peak)
    got = TR._collect(steps, out_dir, raw["vocab"])
    ref = {rid: P.forward(raw, w, toks) for rid, toks in reqs.items()}
    _compare(got, ref, dt, f"trace replay, {dtype}")
