"""The Nazorax design's configuration, schedule, tensor names and cache needs, and the plain
implementation's own mechanisms worked out by hand (no GPU)."""
import copy
import math

import pytest
import torch

import helpers as H
import nazorax_plain as P
from binfer_b200.cache.manager import CacheManager, KVNeed
from binfer_b200.config import (ConfigError, ConvWindowAttentionSpec, GatedMLPSpec,
                                LatentAttentionSpec, MoESpec, NazoraxConfig, parse_config)
from binfer_b200.parts.base import BuildEnv
from binfer_b200.parts.model import DecoderModel, param_specs_for

CPU = BuildEnv(torch.float32, torch.device("cpu"))
F64 = torch.float64


def test_the_registry_picks_the_family_by_its_one_name():
    cfg = parse_config(H.NAZ_A)
    assert isinstance(cfg, NazoraxConfig)
    assert cfg.to_dict() == H.NAZ_A and cfg.to_dict() is not H.NAZ_A


def test_layers_become_specs_with_their_own_sizes():
    spec = NazoraxConfig.from_dict(H.NAZ_A).to_spec()
    assert spec.hidden_size == 64 and spec.vocab_size == 300 and not spec.tie_word_embeddings
    assert spec.final_norm.kind == "tanh_norm" and spec.final_norm.bias_suffix == ".b"
    assert spec.pass_projection == "loop.in" and spec.pass_table is None
    assert all(l.block == "parallel" and l.norm.kind == "tanh_norm" for l in spec.layers)
    a, l1, l2 = [l.mixer for l in spec.layers]
    assert isinstance(a, ConvWindowAttentionSpec) and a.proj_bias
    assert (a.num_heads, a.num_kv_heads, a.head_dim, a.value_dim, a.window, a.scale) == (
        4, 2, 32, 16, 24, 0.3)
    assert (a.conv_taps, a.unit_norm, a.proj_norm, a.sinks, a.keep_first) == (0, False, False, False, 0)
    assert a.position.rotary_dim == 20 and a.position.layout == "half" and a.position.ramp_scaling is None
    assert isinstance(l1, LatentAttentionSpec) and l1.sinks and not l1.head_gate and l1.q_rank == 0
    assert (l1.num_heads, l1.head_dim, l1.rot_dim, l1.value_dim, l1.kv_rank, l1.scale) == (
        3, 24, 8, 20, 40, 0.2) and l1.norm_eps == 1e-5
    r = l1.position.ramp_scaling
    assert (r.factor, r.original, r.fast, r.slow, r.magnitude) == (4.0, 64.0, 8.0, 1.0, None)
    assert l1.position.layout == "half" and l2.position.theta == 500.0
    f, m = spec.layers[0].ffn, spec.layers[1].ffn
    assert isinstance(f, GatedMLPSpec) and f.bias and f.activation == "silu"
    assert f.intermediate_size == 96 and f.bias_names == ("gate.b", "up.b", "down.b")
    assert isinstance(m, MoESpec) and m.activation == "clamped" and m.scoring == "softmax_top"
    assert (m.num_experts, m.top, m.expert_size, m.limit, m.shared_size, m.shared_limit) == (
        8, 2, 32, 1.5, 48, 0.7) and not m.shared_gate and (m.slope, m.up_offset) == (1.702, 1.0)
    assert spec.layers[2].ffn is None
    b = NazoraxConfig.from_dict(H.NAZ_B).to_spec()
    assert b.layers[1].ffn.shared_size == 0 and b.layers[0].mixer.position.ramp_scaling is None


def test_the_schedule_repeats_the_loop_and_projects_before_every_pass():
    def runs(raw):
        return [(e.layer, e.before is not None and e.before.project, e.cache_from)
                for e in NazoraxConfig.from_dict(raw).schedule()]
    assert runs(H.NAZ_A) == [(0, True, None), (1, False, None), (0, True, None), (1, False, None),
                             (2, False, None)]
    assert runs(H.NAZ_B) == [(0, False, None)] + 3 * [(1, True, None), (2, False, None)] + [
        (3, False, None)]
    assert runs(H.NAZ_C) == [(0, False, None), (1, False, None), (2, False, None)]
    for raw in (H.NAZ_A, H.NAZ_B, H.NAZ_C, H.NAZ_D):
        assert [(l, p) for l, p, _ in runs(raw)] == P.layer_order(raw)
    spec = NazoraxConfig.from_dict(H.NAZ_C).to_spec()
    assert spec.pass_projection is None


def test_tensor_names_and_shapes():
    shapes = {s.name: s.shape for s in param_specs_for(NazoraxConfig.from_dict(H.NAZ_A).to_spec())}
    assert shapes["embed"] == shapes["head"] == (300, 64) and shapes["loop.in"] == (64, 128)
    for n in ("final.norm", "l0.norm1", "l2.norm1"):
        assert shapes[n] == shapes[n + ".b"] == (64,) and shapes[n + ".alpha"] == ()
    assert not any("norm2" in n for n in shapes)
    assert shapes["l0.mix.q"] == (128, 64) and shapes["l0.mix.q.b"] == (128,)
    assert shapes["l0.mix.k"] == (64, 64) and shapes["l0.mix.k.b"] == (64,)
    assert shapes["l0.mix.v"] == (32, 64) and shapes["l0.mix.v.b"] == (32,)
    assert shapes["l0.mix.o"] == (64, 64) and "l0.mix.o.b" not in shapes
    assert shapes["l0.mlp.gate"] == shapes["l0.mlp.up"] == (96, 64)
    assert shapes["l0.mlp.gate.b"] == shapes["l0.mlp.up.b"] == (96,)
    assert shapes["l0.mlp.down"] == (64, 96) and shapes["l0.mlp.down.b"] == (64,)
    assert shapes["l1.mix.q"] == (3 * 32, 64) and shapes["l1.mix.dkv"] == (48, 64)
    assert shapes["l1.mix.dkv.norm"] == (40,) and shapes["l1.mix.uk"] == (72, 40)
    assert shapes["l1.mix.uv"] == (60, 40) and shapes["l1.mix.sink"] == (3,)
    assert shapes["l1.mix.o"] == (64, 60) and "l1.mix.g" not in shapes and "l1.mix.q.b" not in shapes
    assert shapes["l1.mlp.router"] == (8, 64) and shapes["l1.mlp.e7.down"] == (64, 32)
    assert shapes["l1.mlp.shared.gate"] == (48, 64) and "l1.mlp.shared.gate.b" not in shapes
    assert "l1.mlp.shared.sg" not in shapes and not any(n.startswith("l2.mlp.") for n in shapes)
    shapes = {s.name: s.shape for s in param_specs_for(NazoraxConfig.from_dict(H.NAZ_C).to_spec())}
    assert "loop.in" not in shapes and "l1.mlp.shared.gate" not in shapes


def test_cache_needs_per_layer_run():
    model = DecoderModel(NazoraxConfig.from_dict(H.NAZ_A).to_spec(), CPU)
    kv = model.kv_needs()
    assert kv[0] == kv[2] == KVNeed(2, 32, 24, 16)          # a cache of its own for every pass
    assert kv[1] == kv[3] == KVNeed(1, 48, None, 0)         # the latent and the shared key part
    assert kv[4] == KVNeed(1, 36, None, 0)
    assert all(s is None for s in model.state_needs())
    cm = CacheManager(kv, model.state_needs(), page_size=8, num_pages=6, max_requests=2)
    assert len(cm.groups) == 3


@pytest.mark.parametrize("bad,msg", [
    (lambda r: r["layers"][0].update(type="delta"), "type"),
    (lambda r: r["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda r: r["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda r: r["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda r: r["layers"][0]["mixer"]["rot"].update(dims=34), "dims"),
    (lambda r: r["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda r: r["layers"][1]["mixer"].pop("rot"), "rot"),
    (lambda r: r["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda r: r["layers"][0]["mlp"].update(kind="sparse"), "kind"),
    (lambda r: r["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda r: r["layers"][1]["mlp"]["router"].update(top=9), "top"),
    (lambda r: r["layers"][1]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda r: r["layers"][1]["mlp"]["shared"].update(limit=-1.0), "limit"),
    (lambda r: r["loop"].update(stop=4), "stop"),
    (lambda r: r["loop"].update(times=0), "times"),
    (lambda r: r.pop("vocab"), "vocab"),
    (lambda r: r.update(layers=[]), "layers"),
    (lambda r: r["norm"].update(eps=0.0), "eps"),
])
def test_a_bad_configuration_is_refused(bad, msg):
    raw = copy.deepcopy(H.NAZ_A)
    bad(raw)
    with pytest.raises(ConfigError, match=msg):
        NazoraxConfig.from_dict(raw)


def test_parts_refuse_what_they_cannot_do():
    from binfer_b200.config.specs import LayerSpec, ModelSpec, PassStart, ScheduleEntry
    from binfer_b200.parts.attention_conv_window import ConvWindowAttention
    from binfer_b200.parts.moe import MoEFeedForward
    with pytest.raises(ValueError, match="convolution"):
        ConvWindowAttention(ConvWindowAttentionSpec(num_heads=1, num_kv_heads=1, head_dim=4,
                                                    value_dim=4, conv_taps=3, proj_bias=True), 8, "m.", CPU)
    with pytest.raises(ValueError, match="limit"):
        MoEFeedForward(MoESpec(num_experts=2, top=1, expert_size=4, activation="clamped"), 8, "f.", CPU)
    spec = NazoraxConfig.from_dict(H.NAZ_C).to_spec()
    import dataclasses
    with pytest.raises(ValueError, match="pass projection"):
        DecoderModel(dataclasses.replace(spec, schedule=(
            ScheduleEntry(0, None, PassStart(project=True)),)), CPU)


def test_a_stacked_weight_counts_once():
    """A parallel layer's two last products are one: the parts keep column blocks of its weight."""
    model = DecoderModel(NazoraxConfig.from_dict(H.NAZ_A).to_spec(), CPU)
    sizes = 0
    for s in model.param_specs():
        n = 1
        for d in s.shape:
            n *= d
        sizes += n
    block = model.blocks[1]
    assert block.stacked
    block.load(lambda s: torch.randn(s.shape) if s.shape else torch.tensor(1.0))
    assert block.mixer.w_out.data_ptr() == block.w_out.data_ptr()
    assert block.ffn.w_out.untyped_storage().data_ptr() == block.w_out.untyped_storage().data_ptr()
    assert block.w_out.shape == (64, 60 + 8 * 32 + 48)
    only = [b for b in model.blocks if b is block]
    model.blocks = only
    n = sum(int(torch.Size(s.shape).numel()) for s in block.param_specs())
    # (alpha is a number on the host)
    assert model.weight_bytes() == 4 * (n - 1)


# ------------------------------------------------- the plain implementation, by hand
def test_plain_rotation_in_halves():
    x = torch.arange(2 * 1 * 6, dtype=F64).view(2, 1, 6) + 1.0
    y = P.rotate_halves(x, {"base": 100.0, "dims": 4})
    assert torch.equal(y[0], x[0]) and torch.equal(y[..., 4:], x[..., 4:])
    c, s = math.cos(1.0), math.sin(1.0)                       # pair 0 at position 1: (7, 9)
    assert abs(float(y[1, 0, 0]) - (7 * c - 9 * s)) < 1e-12
    assert abs(float(y[1, 0, 2]) - (9 * c + 7 * s)) < 1e-12
    c, s = math.cos(0.1), math.sin(0.1)                       # pair 1: 100^(-2/4)
    assert abs(float(y[1, 0, 1]) - (8 * c - 10 * s)) < 1e-12


def test_plain_stretched_frequencies():
    """Eight sizes, base e^2: the index of a wave that makes t turns over 2 pi e^2 positions is
    8 (2 - ln t) / 4.  With fast = e and slow = 1: lo = 2, hi = 4."""
    base, original = math.exp(2.0), 2 * math.pi * math.exp(2.0)
    f, mag = P.frequencies({"base": base, "dims": 8, "scaling": {
        "factor": 5.0, "original": original, "fast": math.exp(1.0) * (1 - 1e-9),
        "slow": 1.0 + 1e-9}})
    plain = [base ** (-2.0 * i / 8) for i in range(4)]
    assert abs(mag - (0.1 * math.log(5.0) + 1.0)) < 1e-12
    for i, r in enumerate((0.0, 0.0, 0.0, 0.5)):              # ramp from 2 to 4
        assert abs(f[i] - (plain[i] / 5.0 * r + plain[i] * (1 - r))) < 1e-12
    assert P.frequencies({"base": base, "dims": 8}) == (plain, 1.0)


def test_plain_window_and_sink():
    """A window of two: the third token back is out.  A sink of ln 2 beside two scores of zero
    takes half of the weight and gives nothing."""
    T = 4
    q, k = torch.ones(T, 1, 2, dtype=F64), torch.zeros(T, 1, 2, dtype=F64)
    v = torch.eye(T, dtype=F64).view(T, 1, T)
    o = P.softmax_attention(q, k, v, 1.0, 2)
    assert o[0, 0].tolist() == [1.0, 0.0, 0.0, 0.0] and o[3, 0].tolist() == [0.0, 0.0, 0.5, 0.5]
    o = P.softmax_attention(q, k, v, 1.0, 2, torch.tensor([math.log(2.0)], dtype=F64))
    assert torch.allclose(o[3, 0], torch.tensor([0.0, 0.0, 0.25, 0.25], dtype=F64), atol=1e-12)
    assert abs(float(o[0, 0, 0]) - 1.0 / 3.0) < 1e-12


def test_plain_clamped_expert_and_router_by_hand():
    w = {"e.gate": torch.tensor([[2.0]]), "e.up": torch.tensor([[1.0]]), "e.down": torch.tensor([[1.0]])}
    w = {n: t.double() for n, t in w.items()}

    def by_hand(g, u):
        return g / (1.0 + math.exp(-1.702 * g)) * (u + 1.0)
    h = torch.tensor([[10.0], [-10.0], [0.25]], dtype=F64)
    got = P.expert(h, w, "e.", 1.5).view(-1).tolist()
    # the gate is cut above only, the other projection on both sides
    for a, b in zip(got, (by_hand(1.5, 1.5), by_hand(-20.0, -1.5), by_hand(0.5, 0.25))):
        assert abs(a - b) < 1e-12
    # two of three experts by the softmax over their own logits; a shared one on top
    one = torch.ones(1, 1, dtype=F64)
    w = {"m.router": torch.tensor([[1.0], [3.0], [2.0]], dtype=F64)}
    for e, p in enumerate(("m.e0.", "m.e1.", "m.e2.", "m.shared.")):
        w.update({p + "gate": one, p + "up": one, p + "down": one * (10.0 ** e)})
    mlp = {"router": {"experts": 3, "top": 2}, "expert": {"limit": 9.0}, "shared": {"limit": 0.5}}
    a = 1.0 / (1.0 + math.exp(-1.0))                          # logits 3 and 2
    want = a * 10.0 * by_hand(1.0, 1.0) + (1 - a) * 100.0 * by_hand(1.0, 1.0) + 1000.0 * by_hand(0.5, 0.5)
    assert abs(float(P.mixture(one, w, "m.", mlp)) - want) < 1e-9


def test_plain_norm_and_bias():
    w = {"n": torch.tensor([2.0, 3.0], dtype=F64), "n.b": torch.tensor([0.5, -0.5], dtype=F64),
         "n.alpha": torch.tensor(0.5, dtype=F64)}
    y = P.tanh_norm(torch.tensor([[2.0, -4.0]], dtype=F64), w, "n")
    assert abs(float(y[0, 0]) - (2.0 * math.tanh(1.0) + 0.5)) < 1e-12
    assert abs(float(y[0, 1]) - (3.0 * math.tanh(-2.0) - 0.5)) < 1e-12


def test_every_constant_and_small_tensor_counts(tmp_path):
    """The plain logits move when the sinks, a bias, alpha, the stretching of the waves, a limit,
    the loop's projection or its repeats are changed: a fault in any of them shows in the whole
    models' tests on the GPU, whose float32 bound is a hundred times smaller."""
    d = H.make_nazorax_dir(tmp_path, "A")
    raw, w = H.read_model_dir(d)
    toks = H.random_tokens(60, raw["vocab"], 4)
    ref = P.forward(raw, w, toks)
    for name in ("l1.mix.sink", "l0.mix.q.b", "l0.mix.k.b", "l0.mix.v.b", "l0.mlp.gate.b", "l0.mlp.up.b",
                 "l0.mlp.down.b", "l0.norm1.b", "final.norm.b", "l1.norm1.alpha", "final.norm.alpha"):
        off = {n: t.clone() for n, t in w.items()}
        off[name] = off[name] * 0.5 if name.endswith("alpha") else torch.zeros_like(off[name])
        if name.endswith("sink"):
            off[name] -= 40.0
        assert H.rel_err(P.forward(raw, off, toks), ref) > 6e-3, name
    off = {n: t.clone() for n, t in w.items()}
    off["loop.in"][:, 64:] = 0.0                              # the embedding output's half
    assert H.rel_err(P.forward(raw, off, toks), ref) > 6e-3
    for change in (lambda r: r["layers"][1]["mixer"]["rot"].pop("scaling"),
                   lambda r: r["layers"][2]["mixer"]["rot"]["scaling"].update(factor=2.0),
                   lambda r: r["layers"][1]["mlp"]["expert"].update(limit=1.4),
                   lambda r: r["layers"][1]["mlp"]["shared"].update(limit=1.5),
                   lambda r: r["layers"][0]["mixer"]["mask"].update(size=23),
                   lambda r: r["layers"][0]["mixer"]["rot"].update(dims=22),
                   lambda r: r["loop"].update(times=1), lambda r: r["loop"].update(stop=1)):
        other = copy.deepcopy(raw)
        change(other)
        assert H.rel_err(P.forward(other, w, toks), ref) > 6e-3
