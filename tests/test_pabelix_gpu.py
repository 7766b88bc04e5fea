"""The Pabelix design on the GPU against its plain implementation.

Each kernel alone (attention with marked keys at the edges of tiles, shares and pages), each
mechanism alone, one-layer models whose weights make one key stand out, then whole models in
every replay regime, both precisions, with page pools so small that every page is used again,
the residual stream after every layer, and generation through the engine's own entry point and
scheduler.
"""
import math

import pytest
import torch

import helpers as H
import pabelix_plain as P

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


def _one_layer(layers, vocab=260, width=48, eps=1e-5):
    return {"architecture": "Pabelix", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": layers}


# ------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("dtype", [torch.float32, BF16], ids=["f32", "bf16"])
@pytest.mark.parametrize("width", [64, 51, 1])
def test_embedding_with_position_vectors(cuda_device, dtype, width):
    """Near and very far positions, even and odd widths, a scale on the table's rows."""
    from binfer_b200.csrc import ops
    g = torch.Generator().manual_seed(width)
    table = torch.randn(20, width, generator=g).to(dtype)
    pos = [0, 1, 2, 77, 4095, 131071, 1000003]
    ids = torch.tensor([3, 0, 19, 7, 7, 1, 2], dtype=torch.int32)
    out = torch.empty(len(pos), width, device=cuda_device)
    i = torch.arange((width + 1) // 2, dtype=F64)
    freqs = 10000.0 ** (-2.0 * i / width)
    ops.embed_gather(table.to(cuda_device), ids.to(cuda_device), out, 0.5,
                     ops.error_word(cuda_device),
                     torch.tensor(pos, dtype=torch.int32, device=cuda_device),
                     freqs.to(cuda_device))
    ang = torch.tensor(pos, dtype=F64)[:, None] * freqs[None]
    vec = torch.zeros(len(pos), width, dtype=F64)
    vec[:, 0::2], vec[:, 1::2] = torch.sin(ang), torch.cos(ang)[:, :width // 2]
    want = table[ids.long()].double() * 0.5 + vec
    assert float((out.cpu().double() - want).abs().max()) <= 1e-6


@pytest.mark.parametrize("dtype", [torch.float32, BF16], ids=["f32", "bf16"])
@pytest.mark.parametrize("width", [8, 51, 320, 1536, 4096, 8192])
def test_norm_of_an_output_with_the_next_norm(cuda_device, dtype, width):
    """One kernel: the norm of a sublayer's output, the add, the next norm of the new stream;
    without a next norm the old result."""
    from binfer_b200.csrc import ops
    g = torch.Generator().manual_seed(width)
    x = torch.randn(5, width, generator=g)
    y = (torch.randn(5, width, generator=g) * 3).to(dtype)
    w, w2 = torch.rand(width, generator=g) + 0.5, torch.rand(width, generator=g) + 0.5
    d = lambda t: t.double()                                     # noqa: E731
    new = d(x) + P.rms_norm(d(y), d(w) - 1.0, 1e-3)
    nxt = P.rms_norm(new, d(w2) - 1.0, 1e-2)
    for with_next in (True, False):
        resid, out = x.to(cuda_device), torch.empty(5, width, dtype=dtype, device=cuda_device)
        ops.rmsnorm_add(resid, y.to(cuda_device), w.to(cuda_device), out, 1e-3,
                        next_weight=w2.to(cuda_device) if with_next else None, next_eps=1e-2)
        assert H.rel_err(resid.cpu(), new) <= 2e-6
        want = nxt if with_next else new
        assert H.rel_err(out.float().cpu(), want) <= (2e-6 if dtype == torch.float32 else 6e-3)


@pytest.mark.parametrize("tokens,inner,width", [(1, 2048, 256), (8, 3072, 512), (64, 2560, 264),
                                                (300, 512, 256), (1100, 520, 256)])
def test_products_with_the_clamped_activation(cuda_device, tokens, inner, width):
    """The stacked product with the activation in its epilogue, for few tokens and for many: the
    same as the product followed by the activation, within the rounding of what lies between."""
    from binfer_b200.csrc import ops
    g = torch.Generator().manual_seed(tokens)
    x = torch.randn(tokens, width, generator=g).to(BF16)
    w = (torch.randn(2 * inner, width, generator=g) * 2 / width ** 0.5).to(BF16)
    limit = 1.25
    eye = torch.eye(inner, dtype=F64)
    want = P.clamped_mlp(x.double(), {"f.gate": w[:inner].double(), "f.up": w[inner:].double(),
                                      "f.down": eye}, "f.", limit)
    out = torch.empty(tokens, inner, dtype=BF16, device=cuda_device)
    k = dict(activation="clamped", limit=limit, slope=1.702, up_offset=1.0)
    xd, wd, err = x.to(cuda_device), w.to(cuda_device), ops.error_word(cuda_device)
    ran = 0
    if tokens <= 64:
        plan = ops.gemm_swiglu_plan(inner, width, cuda_device)
        assert plan and ops.gemm_bf16_swiglu(xd, wd, out, err, plan[0], **k)
        assert H.rel_err(out.float().cpu(), want) <= 6e-3
        ran += 1
    if tokens >= 64:
        out.zero_()
        assert ops.gemm_bf16_pair(xd, wd, out, err, gated=True, **k)
        assert H.rel_err(out.float().cpu(), want) <= 6e-3
        ran += 1
    assert ran and int(err.item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, BF16], ids=["f32", "bf16"])
@pytest.mark.parametrize("inner,limit", [(64, 1.5), (13, 0.3), (256, 7.0)])
def test_clamped_activation(cuda_device, dtype, inner, limit):
    from binfer_b200.csrc import ops
    g = torch.Generator().manual_seed(inner)
    gu = (torch.randn(9, 2 * inner, generator=g) * 3).to(dtype)
    gu[0, :4] = torch.tensor([limit, 50.0, -50.0, 0.0]).to(dtype)
    gu[0, inner:inner + 4] = torch.tensor([-50.0, 50.0, limit, -limit]).to(dtype)
    out = torch.empty(9, inner, dtype=dtype, device=cuda_device)
    ops.gated_act_mul(gu.to(cuda_device), out, "clamped", limit, 1.702, 1.0)
    eye = torch.eye(inner, dtype=F64)
    z = torch.zeros(inner, inner, dtype=F64)
    want = P.clamped_mlp(gu.double(), {"f.gate": torch.cat([eye, z], 1),
                                       "f.up": torch.cat([z, eye], 1), "f.down": eye}, "f.", limit)
    assert H.rel_err(out.float().cpu(), want) <= (2e-6 if dtype == torch.float32 else 6e-3)


@pytest.mark.parametrize("experts,groups,keep,top,T", [
    (8, 2, 1, 2, 40), (6, 1, 1, 2, 40), (5, 5, 3, 2, 40), (64, 8, 3, 6, 40), (9, 3, 2, 4, 700),
    (1, 1, 1, 1, 40), (12, 4, 4, 12, 40), (96, 2, 2, 8, 40)])
def test_router_of_sigmoid_scores(cuda_device, experts, groups, keep, top, T):
    """Choices and weights against the plain router; with groups of more than two experts the
    choice differs from that of groups counted by their best expert alone."""
    from binfer_b200.csrc import ops
    g = torch.Generator().manual_seed(experts * 10 + groups)
    width = 40
    h = torch.randn(T, width, generator=g)
    wr = torch.randn(experts, width, generator=g) * 0.3
    router = {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}
    ids, wts = P.route(h.double(), {"r.router": wr.double()}, "r.", router)
    route_w = torch.empty(T, experts, device=cuda_device)
    top_ids = torch.empty(T, top, dtype=torch.int32, device=cuda_device)
    top_w = torch.empty(T, top, device=cuda_device)

    def run(group_top):
        ops.moe_route(h.to(cuda_device), wr.to(cuda_device), experts, top, False, route_w, top_ids,
                      top_w, scoring="sigmoid", groups=groups, groups_keep=keep,
                      group_top=group_top, normalize=False)
        return top_ids.cpu().long().sort(-1).values

    ones = run(1)
    got = run(2)
    want = torch.zeros(T, experts, dtype=F64).scatter_(1, ids, wts)
    same = (got == ids.sort(-1).values).all(-1)
    assert int((~same).sum()) <= T // 40                 # (two nearly equal scores)
    assert H.rel_err(route_w.cpu()[same], want[same]) <= 2e-6
    assert H.rel_err(top_w.cpu().sum(-1)[same], wts.sum(-1)[same]) <= 2e-6
    if 1 < groups and keep < groups and experts // groups > 2:
        assert not torch.equal(ones, got)


# ------------------------------------------------------------- the attention kernels alone
SIZES = {  # heads, kv heads, d, dv
    "tcgen05": (4, 2, 64, 128), "tcgen05_one": (3, 3, 64, 128), "tcgen05_many": (16, 2, 64, 128),
    "pair64": (6, 3, 32, 64), "mma": (4, 2, 48, 96), "mma_wide": (2, 1, 128, 128),
    "mma_small": (5, 5, 16, 16), "mma_many": (40, 2, 16, 32), "mma_tall": (3, 1, 16, 112),
    "odd": (3, 1, 7, 5), "large": (2, 1, 200, 300)}


class _Case:
    """Requests with cached tokens and new ones at the end, pages in a shuffled order, keys and
    values stored by the engine's own kernel; q, k, v and the gate are column blocks of one row a
    token, as the stacked product leaves them."""

    def __init__(self, dev, sizes, dtype, page_size, ctx, q_lens, temp=(0.4, 16), seed=0,
                 spike=None):
        from binfer_b200.csrc import ops
        self.dev, self.dtype, self.ps = dev, dtype, page_size
        self.nh, self.nkv, self.d, self.dv = sizes
        nh, nkv, d, dv = sizes
        g = torch.Generator().manual_seed(seed)
        self.ctx, self.q_lens = ctx, q_lens
        self.scale, self.lam, self.eps, self.factor = d ** -0.5, 0.7, 1e-5, 0.6
        self.temp = {"coef": temp[0], "every": temp[1]} if temp else None
        cols = [nh * 2 * d, nkv * 2 * d, nkv * dv, nh * dv]
        self.offs = [0, cols[0], sum(cols[:2]), sum(cols[:3])]
        width = sum(cols)
        self.rows = [torch.randn(n, width, generator=g) for n in ctx]
        self.spike = spike
        if spike is not None:              # (request, query, key, map): one score stands out
            b, i, j, m = spike
            for h in range(nh):
                at = h * 2 * d + m * d
                v = torch.randn(d, generator=g) + 0.5
                v = v / v.norm() * (math.sqrt(d) * 3.0)
                self.rows[b][i, at:at + d] = v
                kv = self.offs[1] + (h // (nh // nkv)) * 2 * d + m * d
                if h % (nh // nkv) == 0:
                    self.rows[b][j, kv:kv + d] = v
        self.rows = [r.to(dtype) for r in self.rows]
        n_pages = [-(-n // page_size) for n in ctx]
        order = (torch.randperm(sum(n_pages), generator=g) + 1).tolist()
        W = max(n_pages)
        tables = torch.zeros(len(ctx), W, dtype=torch.int32)
        at = 0
        for b, n in enumerate(n_pages):
            tables[b, :n] = torch.tensor(order[at:at + n], dtype=torch.int32)
            at += n
        self.tables = tables.to(dev)
        pages = sum(n_pages) + 1
        self.k = torch.zeros(pages, nkv, page_size, 2 * d, dtype=dtype, device=dev)
        self.v = torch.zeros(pages, nkv, page_size, dv, dtype=dtype, device=dev)
        self.err = ops.error_word(dev)
        slots = [int(tables[b, p // page_size]) * page_size + p % page_size
                 for b, n in enumerate(ctx) for p in range(n)]
        ops.kv_store(torch.cat(self.rows).to(dev), self.offs[1], self.offs[2],
                     torch.tensor(slots, dtype=torch.int32, device=dev), self.k, self.v, self.err)
        new = [r[n - q:] for r, n, q in zip(self.rows, ctx, q_lens)]
        self.proj = torch.cat(new).to(dev)
        i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)       # noqa: E731
        self.positions = i32([p for n, q in zip(ctx, q_lens) for p in range(n - q, n)])
        self.seq = i32([b for b, q in enumerate(q_lens) for _ in range(q)])
        self.items = i32([[b, sum(q_lens[:b]), q, ctx[b] - q] for b, q in enumerate(q_lens)])
        self.q = self.proj[:, :nh * 2 * d]
        self.gate = self.proj[:, self.offs[3]:]

    def combine(self, gate=True):
        from binfer_b200.csrc import ops
        t = self.temp or {"coef": 0.0, "every": 1}
        return ops.DiffCombine(self.lam, self.eps, self.factor, self.gate if gate else None,
                               t["coef"], t["every"])

    def run(self, kind, variant=None, splits=0, gate=True):
        from binfer_b200.csrc import ops
        out = torch.full((self.proj.shape[0], self.nh * self.dv), float("nan"), dtype=self.dtype,
                         device=self.dev)
        dc = self.combine(gate)
        if kind == "generic":
            ops.diff_attention_generic(self.q, self.k, self.v, self.seq, self.positions,
                                       self.tables, out, self.nh, self.scale, dc, self.err)
        elif kind == "decode":
            ops.diff_attention_decode(self.q, self.k, self.v, None, self.proj.shape[0], self.seq,
                                      self.positions, self.tables, out, self.nh, self.scale, dc,
                                      max(self.ctx), self.err, variant=variant)
        else:
            ops.diff_attention_prefill(self.q, self.k, self.v, self.items, len(self.ctx),
                                       max(self.q_lens), self.tables, out, self.nh, self.scale,
                                       dc, self.err, max_ctx=max(self.ctx), variant=variant,
                                       splits=splits)
        assert int(self.err.item()) == 0
        return out.float().cpu()

    def plain(self, gate=True, lam=None, swap=None):
        """``swap``: (request, key) whose key row of both maps is zeroed (what a kernel that
        misses it would see, nearly)."""
        nh, nkv, d, dv = self.nh, self.nkv, self.d, self.dv
        out = []
        for b, r in enumerate(self.rows):
            T, r = r.shape[0], r.double()
            q = r[:, :self.offs[1]].view(T, nh, 2, d) * P.query_temperature(T, self.temp)[:, None, None, None]
            k = r[:, self.offs[1]:self.offs[2]].reshape(T, nkv, 2, d).clone()
            if swap is not None and swap[0] == b:
                k[swap[1]] = 0.0
            v = r[:, self.offs[2]:self.offs[3]].reshape(T, nkv, dv)
            o = torch.zeros(T, nh, dv, dtype=F64)
            for h in range(nh):
                g = h // (nh // nkv)
                a = [P.softmax_map(q[:, h, m], k[:, g, m], v[:, g], self.scale) for m in (0, 1)]
                # (combine_maps' last factor is 1 - diff)
                o[:, h] = P.combine_maps(a[0], a[1], self.lam if lam is None else lam,
                                         1.0 - self.factor, self.eps)
            o = o.reshape(T, nh * dv)
            if gate:
                o = o * torch.sigmoid(r[:, self.offs[3]:])
            out.append(o[T - self.q_lens[b]:])
        return torch.cat(out)


def _kernels(sizes, page_size, single):
    """(kind, variant) of every kernel that takes these sizes."""
    nh, nkv, d, dv = sizes
    out = [("generic", None)]
    if d % 16 == 0 and dv % 16 == 0 and d <= 128 and dv <= 128:
        out.append(("prefill", "mma_sync"))
        if (d, dv) == (64, 128) and 8 <= page_size <= 64:
            out.append(("prefill", "umma"))
        if single:
            out.append(("decode", "mma_sync"))
            if 2 * d == dv and dv in (64, 128) and page_size >= 8 and nh // nkv <= 8:
                out.append(("decode", "persistent"))
    return out


CTX = {"portions": ([70, 130, 1, 300], [70, 2, 1, 200]), "single": ([1, 64, 65, 128, 129, 400], [1] * 6)}


@pytest.mark.parametrize("page_size", [16, 64, 4])
@pytest.mark.parametrize("what", sorted(CTX))
@pytest.mark.parametrize("name", sorted(SIZES))
def test_attention_kernels(cuda_device, name, what, page_size):
    """Every kernel that takes the sizes, bfloat16 and float32, unequal requests in one launch."""
    sizes = SIZES[name]
    ctx, q_lens = CTX[what]
    c32 = _Case(cuda_device, sizes, torch.float32, page_size, ctx, q_lens, seed=1)
    assert H.rel_err(c32.run("generic"), c32.plain()) <= 1e-5
    c = _Case(cuda_device, sizes, BF16, page_size, ctx, q_lens, seed=2)
    want = c.plain()
    ran = _kernels(sizes, page_size, what == "single")
    for kind, variant in ran:
        e = H.rel_err(c.run(kind, variant), want)
        assert e <= 1.5e-2, f"{kind} {variant}: {e:.3g}"
    if name.startswith("tcgen05") and page_size >= 8:
        assert ("prefill", "umma") in ran


@pytest.mark.parametrize("m", [0, 1])
@pytest.mark.parametrize("name", ["tcgen05", "pair64", "mma", "odd"])
@pytest.mark.parametrize("key", [0, 1, 31, 32, 63, 64, 127, 128, 129, 255, 256, 398, 399])
def test_a_marked_key_on_every_kernel(cuda_device, name, key, m):
    """One key of one map stands out for the last query, at the edges of pages, of key tiles, of
    shares of 128 keys, at the start and beside the query; without it the result is another."""
    sizes = SIZES[name]
    for dtype in (torch.float32, BF16):
        for ctx, q_lens in (([400, 30], [1, 1]), ([400, 30], [150, 30])):
            c = _Case(cuda_device, sizes, dtype, 16, ctx, q_lens, seed=key + m, temp=None,
                      spike=(0, 399, key, m))
            want = c.plain()
            at = q_lens[0] - 1
            moved = H.rel_err(c.plain(swap=(0, key))[at], want[at])
            assert moved > 0.3, f"the key moves its query by {moved:.3g} only"
            for kind, variant in _kernels(sizes, 16, q_lens[0] == 1):
                if dtype == torch.float32 and kind != "generic":
                    continue
                got = c.run(kind, variant)
                e = H.rel_err(got[at], want[at])
                assert e <= (1e-5 if dtype == torch.float32 else 2e-2), f"{kind} {variant}: {e:.3g}"


@pytest.mark.parametrize("m", [0, 1])
@pytest.mark.parametrize("name", ["tcgen05", "pair64", "mma"])
@pytest.mark.parametrize("key", [5, 70, 130, 200, 390])
def test_a_score_that_dwarfs_the_tiles_before_it(cuda_device, name, key, m):
    """A score hundreds above everything before it in one map: what the earlier tiles left in
    that map's output counts nothing any more; the other map's is untouched."""
    sizes = SIZES[name]
    for q_lens in ([1, 1], [150, 30]):
        c = _Case(cuda_device, sizes, BF16, 16, [400, 30], q_lens, seed=key, temp=None,
                  spike=(0, 399, key, m))
        c.scale *= 12.0
        want, at = c.plain(), q_lens[0] - 1
        for kind, variant in _kernels(sizes, 16, q_lens[0] == 1):
            e = H.rel_err(c.run(kind, variant)[at], want[at])
            assert e <= 2e-2, f"{kind} {variant}: {e:.3g}"


@pytest.mark.parametrize("splits", [1, 2, 3, 8])
def test_keys_of_a_portion_shared_out(cuda_device, splits):
    """A few rows after many cached keys on the tcgen05 kernel, the keys shared out over several
    CTAs, some of which have none of a short request's keys; with and without a gate."""
    c = _Case(cuda_device, SIZES["tcgen05"], BF16, 16, [900, 70, 5], [130, 60, 5], seed=3)
    for gate in (True, False):
        e = H.rel_err(c.run("prefill", "umma", splits=splits, gate=gate), c.plain(gate=gate))
        assert e <= 1.5e-2, f"{e:.3g}"


def test_second_map_and_temperature_count(cuda_device):
    """Leaving out the second map, or the query temperature, is another function; the kernels
    compute the full one."""
    sizes = SIZES["mma"]
    c = _Case(cuda_device, sizes, torch.float32, 16, [90, 40], [90, 40], seed=4, temp=(0.8, 7))
    want = c.plain()
    assert H.rel_err(c.plain(lam=0.0), want) > 0.1
    temp, c.temp = c.temp, None
    assert H.rel_err(c.plain(), want) > 0.1
    c.temp = temp
    assert H.rel_err(c.run("generic"), want) <= 1e-5


@pytest.mark.parametrize("kind,variant", [("decode", "mma_sync"), ("decode", "persistent")])
def test_decode_rows_out_of_a_mixed_step(cuda_device, kind, variant):
    """Single tokens named by their rows, between portions that the kernel must leave alone."""
    from binfer_b200.csrc import ops
    c = _Case(cuda_device, SIZES["pair64"], BF16, 16, [50, 200, 33, 140], [7, 1, 3, 1], seed=5)
    rows = torch.tensor([7, 11], dtype=torch.int32, device=cuda_device)
    out = torch.full((12, c.nh * c.dv), 5.0, dtype=BF16, device=cuda_device)
    ops.diff_attention_decode(c.q, c.k, c.v, rows, 2, c.seq, c.positions, c.tables, out, c.nh,
                              c.scale, c.combine(), 200, c.err, variant=variant)
    assert int(c.err.item()) == 0
    got, want = out.float().cpu(), c.plain()
    assert H.rel_err(got[[7, 11]], want[[7, 11]]) <= 1.5e-2
    rest = [i for i in range(12) if i not in (7, 11)]
    assert bool((got[rest] == 5.0).all())


@pytest.mark.parametrize("dtype", [torch.float32, BF16], ids=["f32", "bf16"])
@pytest.mark.parametrize("kv_heads,dk,dv,page_size", [(2, 32, 24, 16), (3, 7, 5, 4), (1, 128, 128, 64)])
def test_keys_and_values_into_the_pages(cuda_device, dtype, kv_heads, dk, dv, page_size):
    from binfer_b200.csrc import ops
    g = torch.Generator().manual_seed(dk)
    T, pages, off = 11, 6, 8
    proj = torch.randn(T, off + kv_heads * (dk + dv) + 3, generator=g).to(dtype)
    k = torch.zeros(pages, kv_heads, page_size, dk, dtype=dtype, device=cuda_device)
    v = torch.zeros(pages, kv_heads, page_size, dv, dtype=dtype, device=cuda_device)
    slots = torch.randperm(pages * page_size, generator=g)[:T].to(torch.int32)
    err = ops.error_word(cuda_device)
    v_off = off + kv_heads * dk
    ops.kv_store(proj.to(cuda_device), off, v_off, slots.to(cuda_device), k, v, err)
    wk, wv = torch.zeros_like(k, device="cpu"), torch.zeros_like(v, device="cpu")
    for t, s in enumerate(slots.tolist()):
        wk[s // page_size, :, s % page_size] = proj[t, off:v_off].view(kv_heads, dk)
        wv[s // page_size, :, s % page_size] = proj[t, v_off:v_off + kv_heads * dv].view(kv_heads, dv)
    assert torch.equal(k.cpu(), wk) and torch.equal(v.cpu(), wv) and int(err.item()) == 0


# ------------------------------------------------------------------ mechanisms alone
def _part(cuda_device, dtype, mlp, width, seed):
    from binfer_b200.config import PabelixConfig
    from binfer_b200.parts.base import BuildEnv, build_ffn
    from binfer_b200.weights import random_tensors
    from binfer_b200.weights.loader import place
    part = build_ffn(PabelixConfig._mlp(mlp, "mlp."), width, "f.", BuildEnv(dtype, cuda_device))
    w = random_tensors(part.param_specs(), seed, 0.1, 0.1, dtype)
    if "f.router" in w:
        w["f.router"] *= 0.1            # scores well below one: no ties between sigmoids
    by_name = {s.name: s for s in part.param_specs()}
    part.load(lambda s: place(w[s.name], by_name[s.name], dtype, cuda_device))
    return part, {n: t.double() for n, t in w.items()}


@pytest.mark.parametrize("dtype", [torch.float32, BF16], ids=["f32", "bf16"])
@pytest.mark.parametrize("mlp,width", [
    (H._pab_moe(8, 2, 32, (2, 1)), 64), (H._pab_moe(6, 3, 16), 48), (H._pab_moe(5, 1, 40, (5, 2)), 50),
    (H._pab_moe(32, 4, 64, (8, 3)), 128), (H._pab_moe(1, 1, 24), 40), (H._pab_dense(96, 0.5), 64),
    (H._pab_dense(13, 2.0), 51)])
def test_feed_forwards_alone(cuda_device, dtype, mlp, width):
    """Many tokens, and one and two (in bfloat16 the chosen experts' rows alone are read)."""
    part, w = _part(cuda_device, dtype, mlp, width, 5)
    g = torch.Generator().manual_seed(width)
    for T in (1, 2, 37):
        h = (torch.randn(T, width, generator=g) * 2).to(dtype)
        got = part.forward(h.to(cuda_device), None)
        e = H.rel_err(got.float().cpu(), P.feed_forward(h.double(), w, "f.", mlp))
        assert e <= (3e-6 if dtype == torch.float32 else 2e-2), f"{T} tokens: {e:.3g}"


def _distinct_tokens(n, vocab, seed):
    return torch.randperm(vocab, generator=torch.Generator().manual_seed(seed))[:n].tolist()


def _stand_out(raw, toks, key, query, m, layer=0, amp=20.0, boost=1.0):
    """The token at ``key`` gets a large part along one direction and the one at ``query`` along
    another; map ``m`` of every key head that ``layer`` reads answers the first with a fixed
    vector, and every query head answers the second with the same vector."""
    mx = raw["layers"][layer]["mixer"]
    src = mx.get("kv_from", layer) if mx.get("kv_from") is not None else layer
    H_, G_, d = mx["heads"], mx["kv_heads"], mx["dim"]

    def tweak(w):
        gen = torch.Generator().manual_seed(9)
        width, dt = w["embed"].shape[1], w["embed"].dtype
        e_k = torch.randn(width, generator=gen)
        e_k = e_k / e_k.norm()
        e_q = torch.randn(width, generator=gen)
        e_q = e_q - (e_q @ e_k) * e_k
        e_q = e_q / e_q.norm()
        a = torch.randn(d, generator=gen)
        a = a / a.norm() * d ** 0.5
        w["embed"][toks[key]] += (e_k * amp).to(dt)
        w["embed"][toks[query]] += (e_q * amp).to(dt)
        for g in range(G_):
            for h in range(g * (H_ // G_), (g + 1) * (H_ // G_)):
                at = (h * 2 + m) * d
                w[f"l{layer}.mix.q"][at:at + d] += (boost * torch.outer(a, e_q)).to(dt)
            at = (g * 2 + m) * d
            w[f"l{src}.mix.k"][at:at + d] += (boost * torch.outer(a, e_k)).to(dt)
        w[f"l{layer}.norm1b"] += 8.0       # the layer's output decides the stream
    return tweak


# pages of 8: the marked key and the query that asks for it; the last 100 of 240 are decoded
EDGES = {"far": (3, 230), "first_token": (0, 235), "page_border": (8, 27), "page_end": (7, 24),
         "second_token": (0, 1), "neighbour": (100, 101), "tile_border": (64, 200),
         "tile_end": (63, 130), "share_border": (128, 239), "share_end": (127, 239),
         "across_the_cut": (130, 150)}


@pytest.mark.parametrize("m", [0, 1])
@pytest.mark.parametrize("case", sorted(EDGES))
def test_attention_layers_with_a_marked_key(cuda_device, tmp_path, case, m):
    """A layer with a cache of its own, and one that reads it: the marked key decides its query's
    logits, in prompts, portions and decoding."""
    key, query = EDGES[case]
    raw = _one_layer([H._pab_layer(H._pab_attn(4, 2, 16, 24, 0.5, scale=0.25)),
                      H._pab_layer(H._pab_attn(4, 2, 16, 24, 0.3, scale=0.25, kv_from=0))],
                     vocab=400)
    toks = _distinct_tokens(240, raw["vocab"], 21)
    d = H.make_pabelix_dir(tmp_path, "A", raw=raw, tag=f"{case}{m}",
                           tweak=_stand_out(raw, toks, key, query, m, layer=m))
    raw, w = H.read_model_dir(d)
    ref = {"a": P.forward(raw, w, toks)}
    other = list(toks)
    other[key] = next(t for t in range(raw["vocab"]) if t not in toks)
    moved = H.rel_err(P.forward(raw, w, other)[query], ref["a"][query])
    assert moved > 1000 * TOL[torch.float32], f"{case}: the key moves the logits by {moved:.3g} only"
    for name, steps in _all_regimes({"a": toks}, tail=100).items():
        got = H.run_trace(_runner(d, torch.float32, 8, H.peak_pages(steps, 8)), steps)
        _compare(got, ref, torch.float32, f"{case}/{name}")


@pytest.mark.parametrize("sizes", ["tcgen05", "pair64", "mma"])
@pytest.mark.parametrize("case", ["far", "first_token", "tile_border", "share_end", "neighbour",
                                  "across_the_cut"])
def test_marked_keys_on_the_tensor_cores(cuda_device, tmp_path, case, sizes):
    """The marked keys again in bfloat16, on the tensor-core kernels and on the kernel for any
    sizes, which on the same rounded numbers is the sharp comparison."""
    from binfer_b200.csrc import ops
    from binfer_b200.parts import attention_diff as mod
    from binfer_b200.profiling import Profiler
    key, query = EDGES[case]
    h, g, dk, dv = SIZES[sizes]
    raw = _one_layer([H._pab_layer(H._pab_attn(h, g, dk, dv, 0.5, scale=4.0 / dk))], vocab=400,
                     width=64)
    toks = _distinct_tokens(240, raw["vocab"], 21)
    d = H.make_pabelix_dir(tmp_path, "D", BF16, raw=raw, tag=case + sizes,
                           tweak=_stand_out(raw, toks, key, query, 0))
    raw, w = H.read_model_dir(d)
    ref = {"a": P.forward(raw, w, toks)}
    other = list(toks)
    other[key] = next(t for t in range(raw["vocab"]) if t not in toks)
    moved = H.rel_err(P.forward(raw, w, other)[query], ref["a"][query])
    assert moved > 0.15, f"{case}: the key moves the logits by {moved:.3g} only"
    outs = []
    for on in (True, False):
        mod.TENSOR_CORES = on
        seen, got = set(), {}
        try:
            for name, steps in _all_regimes({"a": toks}, tail=100).items():
                prof = Profiler()
                got[name] = H.run_trace(_runner(d, BF16, 16, H.peak_pages(steps, 16)), steps)
                prof.stop()
                seen |= set(prof.collect())
                at_query = H.rel_err(got[name][("a", query)], ref["a"][query])
                assert at_query <= 0.3 * moved, (
                    f"{case}/{name} (tensor cores {on}): {at_query:.3g} where the key moves {moved:.3g}")
        finally:
            ops.set_profiler(None)
            mod.TENSOR_CORES = True
        want = {"tcgen05": {"diff_attention_prefill_umma", "diff_attention_decode_persistent"},
                "pair64": {"diff_attention_prefill_mma", "diff_attention_decode_persistent"},
                "mma": {"diff_attention_prefill_mma", "diff_attention_decode_mma"}}[sizes]
        used = {s for s in seen if s.startswith("diff_attention")}
        assert used == (want if on else {"diff_attention_generic"}), used
        outs.append(got)
    for name in outs[0]:
        worst = max(H.rel_err(outs[0][name][k], outs[1][name][k]) for k in outs[0][name])
        assert worst <= 0.03, f"{case}/{name}: the kernels differ by {worst:.3g}"


@pytest.mark.parametrize("every,coef", [(1, 0.3), (16, 0.9), (7, 2.0), (1000, 0.5)])
def test_query_temperature_at_its_steps(cuda_device, tmp_path, every, coef):
    """Factors that change at every position, at a page's border, inside pages, or never within
    the sequence; a factor that steps one position late would show."""
    raw = _one_layer([H._pab_layer(H._pab_attn(2, 1, 16, 16, 0.5, scale=0.6, temp=(coef, every)))])
    d = H.make_pabelix_dir(tmp_path, "A", raw=raw, tag=f"t{every}")
    raw, w = H.read_model_dir(d)
    toks = H.random_tokens(120, raw["vocab"], 12)
    ref = {"a": P.forward(raw, w, toks)}
    if every < 120:
        off = _one_layer([H._pab_layer(H._pab_attn(2, 1, 16, 16, 0.5, scale=0.6, temp=None))])
        assert H.rel_err(P.forward(off, w, toks), ref["a"]) > 100 * TOL[torch.float32]
    for name, steps in _all_regimes({"a": toks}, tail=60).items():
        got = H.run_trace(_runner(d, torch.float32, 8, H.peak_pages(steps, 8)), steps)
        _compare(got, ref, torch.float32, f"temperature/{name}")


def test_a_reading_layer_reads_the_layer_it_names(cuda_device, tmp_path):
    """Three caches; two readers.  Reading the neighbouring layer's cache instead moves the
    logits, so the layer named is the one that was read."""
    mk = lambda src: _one_layer([H._pab_layer(H._pab_attn(4, 2, 16, 24)) for _ in range(3)] +   # noqa: E731
                                [H._pab_layer(H._pab_attn(4, 2, 16, 24, kv_from=s)) for s in src])
    raw = mk((0, 2))
    d = H.make_pabelix_dir(tmp_path, "A", raw=raw, tag="readers")
    raw, w = H.read_model_dir(d)
    toks = H.random_tokens(90, raw["vocab"], 12)
    ref = {"a": P.forward(raw, w, toks)}
    for src in ((1, 2), (0, 1), (2, 0)):
        assert H.rel_err(P.forward(mk(src), w, toks), ref["a"]) > 100 * TOL[torch.float32]
    for name, steps in _all_regimes({"a": toks}, tail=40).items():
        got = H.run_trace(_runner(d, torch.float32, 8, H.peak_pages(steps, 8)), steps)
        _compare(got, ref, torch.float32, f"readers/{name}")


# ----------------------------------------------------------------------- whole models
LENGTHS = {"A": [5, 17, 33, 70, 121], "B": [1, 9, 40, 70, 101], "C": [3, 30, 64, 47, 2],
           "D": [2, 45, 150, 300, 90]}


def _requests(which, extra=()):
    vocab = H.PAB[which]["raw"]["vocab"]
    lens = list(LENGTHS[which]) + list(extra)
    return {f"r{i}": H.random_tokens(n, vocab, 100 * i + n) for i, n in enumerate(lens)}


@pytest.fixture(scope="module")
def plain_logits(tmp_path_factory):
    cache = {}

    def get(which, dtype, reqs):
        d = H.make_pabelix_dir(tmp_path_factory.getbasetemp(), which, dtype)
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
                         ids=["A-f32", "B-f32", "C-f32", "D-f32", "A-bf16", "B-bf16", "C-bf16",
                              "D-bf16"])
@pytest.mark.parametrize("regime", ["whole", "tail", "portions", "mixed"])
def test_replay(cuda_device, plain_logits, which, dtype, regime):
    """Seven requests through four request slots and page pools of exactly the peak need."""
    reqs = _requests(which, (55, 61) if regime == "mixed" else ())
    model_dir, ref = plain_logits(which, dtype, reqs)
    steps = _all_regimes(reqs)[regime]
    ps = H.PAB[which]["page_size"]
    runner = _runner(model_dir, dtype, ps, H.peak_pages(steps, ps))
    got = H.run_trace(runner, steps)
    assert not runner.cache.requests and all(g.pool.num_held == 0 for g in runner.cache.groups)
    _compare(got, ref, dtype, f"{which}/{regime}")


@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
def test_the_stream_after_every_layer(cuda_device, plain_logits, which):
    from binfer_b200.engine.runner import StepItem
    toks = H.random_tokens(19, H.PAB[which]["raw"]["vocab"], 77)
    model_dir, _ = plain_logits(which, torch.float32, {})
    raw, w = H.read_model_dir(model_dir)
    want = []
    P.forward(raw, w, toks, want)
    runner = _runner(model_dir, torch.float32, 8, 4)
    runner.add_request("a")
    items = [StepItem("a", toks, [len(toks) - 1])]
    runner.reserve(items)
    ctx = runner.build_context(items)
    ctx.scratch["layer_outputs"] = []
    runner.model.forward(ctx, runner.views)
    got = ctx.scratch["layer_outputs"]
    assert len(got) == len(want) == len(runner.model.spec.schedule)
    for i, (g, r) in enumerate(zip(got, want)):
        assert H.rel_err(g.cpu(), r) <= 2e-5, f"{which}: after layer {i}"


@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
def test_regimes_agree_bitwise_in_float32(cuda_device, plain_logits, which):
    """Every sum's order depends on positions and sizes alone: cutting and batching change
    no bit."""
    reqs = _requests(which)
    model_dir, _ = plain_logits(which, torch.float32, reqs)
    ps = H.PAB[which]["page_size"]
    outs = []
    for steps in _all_regimes(reqs).values():
        outs.append(H.run_trace(_runner(model_dir, torch.float32, ps, H.peak_pages(steps, ps)),
                                steps))
    for other in outs[1:]:
        for key, row in outs[0].items():
            assert torch.equal(row, other[key]), f"{which}: logits at {key} depend on the cut"


@pytest.mark.parametrize("dtype", [torch.float32, BF16], ids=["f32", "bf16"])
def test_long_decoding(cuda_device, plain_logits, dtype):
    """A short prompt, then 300 tokens one by one, over shares of 128 keys."""
    which = "D"
    reqs = {"long": H.random_tokens(304, H.PAB[which]["raw"]["vocab"], 7)}
    model_dir, ref = plain_logits(which, dtype, reqs)
    steps = H.trace_decode_tail(reqs, tail=300)
    runner = _runner(model_dir, dtype, 16, 19)
    _compare(H.run_trace(runner, steps), ref, dtype, "long decoding")


@pytest.mark.parametrize("which,dtype", [("A", torch.float32), ("D", BF16)], ids=["A-f32", "D-bf16"])
def test_decoding_from_captured_steps(cuda_device, plain_logits, which, dtype):
    """Steps of single tokens replayed from CUDA graphs (padded rows use the scratch page)
    give what eager steps give."""
    reqs = _requests(which, (55, 61))
    model_dir, ref = plain_logits(which, dtype, reqs)
    steps = H.trace_mixed(reqs, tail=20)
    ps = H.PAB[which]["page_size"]
    runner = _runner(model_dir, dtype, ps, H.peak_pages(steps, ps))
    runner.enable_decode_graphs(max_batch=4, max_seq_len=512)
    got = H.run_trace(runner, steps)
    assert getattr(runner, "graph_replays", 0) > 0
    _compare(got, ref, dtype, "captured decode steps")


# ------------------------------------------------------------------------- generation
@pytest.mark.parametrize("graphs,step_tokens", [(True, 2048), (False, 7)],
                         ids=["graphs", "portions"])
def test_greedy_generation_through_the_engine(cuda_device, tmp_path, graphs, step_tokens):
    """Prompts of 5/17/33/2 tokens through ``Engine.generate``: the scheduler's admission,
    portions of at most seven tokens beside decoding (second case), captured decode steps
    (first case); every token is the plain implementation's choice."""
    from binfer_b200 import Engine
    d = H.make_pabelix_dir(tmp_path, "A")
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
    """``bin/binfer``'s entry point: the registry picks the family from config.json; greedy
    tokens are the plain implementation's, and sampling with a seed gives the same tokens
    twice."""
    from binfer_b200.cli import main
    d = H.make_pabelix_dir(tmp_path, "C")
    raw, w = H.read_model_dir(d)
    prompt = H.random_tokens(9, raw["vocab"], 3)
    ids = ",".join(map(str, prompt))
    rc = main([d, "--prompt-ids", ids, "--max-tokens", "5", "--dtype", "fp32", "--ignore-eos",
               "-q", "--kv-pages", "32"])
    assert rc == 0
    out = [int(t) for t in capsys.readouterr().out.split()]
    assert len(out) == 5
    logits = P.forward(raw, w, list(prompt) + out)
    for n, tok in enumerate(out):
        row = logits[len(prompt) - 1 + n]
        assert float(row[tok]) >= float(row.max()) - 1e-4 * float(row.abs().max())
    sampled = []
    for _ in range(2):
        rc = main([d, "--prompt-ids", ids, "--max-tokens", "8", "--dtype", "fp32", "--ignore-eos",
                   "-q", "--kv-pages", "32", "--temperature", "0.9", "--seed", "5"])
        assert rc == 0
        sampled.append(capsys.readouterr().out.split())
    assert sampled[0] == sampled[1] and len(sampled[0]) == 8


def test_trace_replay_tool_with_four_requests(cuda_device, tmp_path):
    """``bin/trace_run`` as a user runs it: six requests, at most four live, and a page pool
    sized by ``--max-tokens``."""
    import test_trace_run_gpu as TR
    d = H.make_pabelix_dir(tmp_path, "B")
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
    TR._replay(d, "float32", steps, out_dir, peak)
    got = TR._collect(steps, out_dir, raw["vocab"])
    ref = {rid: P.forward(raw, w, toks) for rid, toks in reqs.items()}
    worst = max(H.rel_err(row, ref[rid][p]) for (rid, p), row in got.items())
    assert got and worst <= TOL[torch.float32], f"worst relative error {worst:.3g}"
