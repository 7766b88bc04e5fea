"""The Pabelix design's configuration, tensor names, cache needs, and the plain implementation's
own mechanisms worked out by hand (no GPU)."""
import copy
import math

import pytest
import torch

import helpers as H
import pabelix_plain as P
from binfer_b200.cache.manager import CacheManager, KVNeed
from binfer_b200.config import (ConfigError, DifferentialAttentionSpec, GatedMLPSpec, MoESpec,
                                PabelixConfig, parse_config)
from binfer_b200.parts.base import BuildEnv
from binfer_b200.parts.model import DecoderModel, param_specs_for

CPU = BuildEnv(torch.float32, torch.device("cpu"))
F64 = torch.float64


def test_the_registry_picks_the_family_by_its_one_name():
    cfg = parse_config(H.PAB_A)
    assert isinstance(cfg, PabelixConfig)
    assert cfg.to_dict() == H.PAB_A and cfg.to_dict() is not H.PAB_A


def test_layers_become_specs_with_their_own_sizes():
    spec = PabelixConfig.from_dict(H.PAB_A).to_spec()
    assert spec.hidden_size == 64 and spec.vocab_size == 300 and spec.tie_word_embeddings
    assert spec.position_vectors.base == 10000.0
    assert spec.final_norm.offset == 1.0 and spec.final_norm.eps == 1e-5
    assert all(l.block == "sandwich" and l.norm.offset == 1.0 for l in spec.layers)
    assert [(e.layer, e.cache_from) for e in spec.schedule] == [(0, None), (1, 0), (2, None),
                                                                (3, 2), (4, 0)]
    a, b, c = [l.mixer for l in spec.layers[:3]]
    assert isinstance(a, DifferentialAttentionSpec)
    assert (a.num_heads, a.num_kv_heads, a.head_dim, a.value_dim) == (4, 2, 16, 24)
    assert (a.scale, a.diff, a.temp_coef, a.temp_every, a.norm_eps) == (0.35, 0.3, 0.25, 8, 1e-5)
    assert a.output_gate and a.own_cache and not b.own_cache and b.diff == 0.6
    assert (c.head_dim, c.value_dim, c.temp_coef, c.temp_every) == (24, 16, 0.4, 5)
    f = spec.layers[0].ffn
    assert isinstance(f, GatedMLPSpec) and f.activation == "clamped"
    assert (f.intermediate_size, f.limit, f.slope, f.up_offset) == (96, 1.5, 1.702, 1.0)
    m = spec.layers[1].ffn
    assert isinstance(m, MoESpec) and m.scoring == "sigmoid" and not m.normalize
    assert (m.num_experts, m.top, m.expert_size, m.groups, m.groups_keep, m.group_top) == (
        8, 3, 32, 4, 2, 2)
    assert (m.shared_size, m.identity, m.correction, m.route_scale) == (0, 0, False, 1.0)
    assert spec.layers[2].ffn.groups == 1 and spec.layers[3].ffn is None
    no_temp = PabelixConfig.from_dict(H.PAB_B).to_spec().layers[0].mixer
    assert no_temp.temp_coef == 0.0


def test_tensor_names_and_shapes():
    shapes = {s.name: s.shape for s in param_specs_for(PabelixConfig.from_dict(H.PAB_A).to_spec())}
    assert shapes["embed"] == (300, 64) and "head" not in shapes and shapes["final.norm"] == (64,)
    for i in range(5):
        assert shapes[f"l{i}.norm1"] == shapes[f"l{i}.norm1b"] == (64,)
    assert shapes["l0.norm2"] == shapes["l0.norm2b"] == (64,)
    assert "l3.norm2" not in shapes and "l3.norm2b" not in shapes
    assert shapes["l0.mix.q"] == (128, 64) and shapes["l0.mix.k"] == (64, 64)
    assert shapes["l0.mix.v"] == (48, 64) and shapes["l0.mix.g"] == (96, 64)
    assert shapes["l0.mix.o"] == (64, 96)
    assert all(shapes[f"l2.mix.{n}"] == (24,) for n in ("lq1", "lk1", "lq2", "lk2"))
    assert "l1.mix.k" not in shapes and "l1.mix.v" not in shapes     # reads layer 0's
    assert shapes["l1.mix.q"] == (128, 64) and shapes["l1.mix.g"] == (96, 64)
    assert shapes["l0.mlp.gate"] == shapes["l0.mlp.up"] == (96, 64)
    assert shapes["l0.mlp.down"] == (64, 96) and shapes["l1.mlp.router"] == (8, 64)
    assert shapes["l1.mlp.e7.gate"] == (32, 64) and shapes["l1.mlp.e7.down"] == (64, 32)
    assert not any(n.startswith("l3.mlp.") for n in shapes)


def test_cache_needs_per_layer():
    """A cached key head is both maps' keys; layers that read another's keep nothing."""
    model = DecoderModel(PabelixConfig.from_dict(H.PAB_A).to_spec(), CPU)
    kv = model.kv_needs()
    assert kv == [KVNeed(2, 32, None, 24), None, KVNeed(1, 48, None, 16), None, None]
    assert all(s is None for s in model.state_needs())
    cm = CacheManager(kv, model.state_needs(), page_size=8, num_pages=6, max_requests=2)
    assert len(cm.groups) == 2
    # keys of both maps as wide as the values: the plain need, without a value size of its own
    wide = DecoderModel(PabelixConfig.from_dict(H.PAB_D).to_spec(), CPU).kv_needs()
    assert wide[0] == KVNeed(2, 128, None, None)


@pytest.mark.parametrize("bad,msg", [
    (lambda r: r["layers"][0].update(type="delta"), "type"),
    (lambda r: r["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda r: r["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda r: r["layers"][0]["mixer"].pop("diff"), "diff"),
    (lambda r: r["layers"][0]["mixer"]["q_temp"].pop("every"), "every"),
    (lambda r: r["layers"][0]["mixer"]["q_temp"].update(every=0), "every"),
    (lambda r: r["layers"][1]["mixer"].update(kv_from=1), "kv_from"),
    (lambda r: r["layers"][1]["mixer"].update(kv_from=2), "kv_from"),
    (lambda r: r["layers"][4]["mixer"].update(kv_from=1), "kv_from"),     # which has none itself
    (lambda r: r["layers"][4]["mixer"].update(kv_from=2), "differ"),
    (lambda r: r["layers"][0]["mlp"].update(kind="other"), "kind"),
    (lambda r: r["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda r: r["layers"][0]["mlp"].update(limit=0.0), "limit"),
    (lambda r: r["layers"][1]["mlp"]["router"]["groups"].update(count=3), "groups"),
    (lambda r: r["layers"][1]["mlp"]["router"]["groups"].update(keep=5), "groups"),
    (lambda r: r["layers"][1]["mlp"]["router"].update(top=5), "top"),
    (lambda r: r["layers"][1]["mlp"].pop("expert"), "expert"),
    (lambda r: r.pop("width"), "width"),
    (lambda r: r["norm"].update(eps=0.0), "eps"),
])
def test_a_bad_configuration_is_refused(bad, msg):
    raw = copy.deepcopy(H.PAB_A)
    bad(raw)
    with pytest.raises(ConfigError, match=msg):
        PabelixConfig.from_dict(raw)


def test_the_learned_number_of_a_layer_and_the_stacked_product():
    from binfer_b200.parts.attention_diff import DifferentialAttention
    spec = DifferentialAttentionSpec(num_heads=2, num_kv_heads=1, head_dim=3, value_dim=5,
                                     scale=0.5, diff=0.25)
    m = DifferentialAttention(spec, 4, "m.", CPU)
    w = {s.name: torch.randn(s.shape, generator=torch.Generator().manual_seed(i))
         for i, s in enumerate(m.param_specs())}
    m.load(lambda s: w[s.name])
    want = (math.exp(float(w["m.lq1"] @ w["m.lk1"])) - math.exp(float(w["m.lq2"] @ w["m.lk2"]))
            + 0.25)
    assert abs(m.lam - want) < 1e-5
    assert torch.equal(m.w_proj, torch.cat([w["m.q"], w["m.k"], w["m.v"], w["m.g"]]))
    assert (m.q_size, m.k_off, m.v_off, m.gate_off) == (12, 12, 18, 23)
    reader = DifferentialAttention(
        DifferentialAttentionSpec(num_heads=2, num_kv_heads=1, head_dim=3, value_dim=5, scale=0.5,
                                  own_cache=False), 4, "m.", CPU)
    assert reader.gate_off == 12 and "m.k" not in [s.name for s in reader.param_specs()]


# ------------------------------------------------- the plain implementation, by hand
def test_plain_position_vectors():
    v = P.position_vectors(3, 5)                     # an odd width ends in a sine
    f1, f2 = 10000.0 ** (-2 / 5), 10000.0 ** (-4 / 5)
    assert v[0].tolist() == [0.0, 1.0, 0.0, 1.0, 0.0]
    want = [math.sin(2.0), math.cos(2.0), math.sin(2 * f1), math.cos(2 * f1), math.sin(2 * f2)]
    assert torch.allclose(v[2], torch.tensor(want, dtype=F64), atol=1e-14)


def test_plain_query_temperature_grows_in_steps():
    """every = 4: the factor is one for the positions 0, 1, 2 and steps at 3, 7, 11."""
    t = P.query_temperature(9, {"coef": 0.5, "every": 4})
    assert t[:3].tolist() == [1.0] * 3
    assert torch.allclose(t[3:7], torch.full((4,), 1 + 0.5 * math.log(2.0), dtype=F64))
    assert torch.allclose(t[7:], torch.full((2,), 1 + 0.5 * math.log(3.0), dtype=F64))
    assert P.query_temperature(3, None).tolist() == [1.0] * 3


def test_plain_difference_of_two_maps():
    """One head, keys of size one.  Map 1 looks at key 0 alone, map 2 weighs both alike."""
    k1, k2 = torch.tensor([[50.0], [-50.0]], dtype=F64), torch.zeros(2, 1, dtype=F64)
    v = torch.tensor([[2.0, 0.0], [0.0, 4.0]], dtype=F64)
    one = torch.ones(2, 1, dtype=F64)
    a1, a2 = P.softmax_map(one, k1, v, 1.0), P.softmax_map(one, k2, v, 1.0)
    assert torch.allclose(a1[1], torch.tensor([2.0, 0.0], dtype=F64))
    assert torch.allclose(a2[1], torch.tensor([1.0, 2.0], dtype=F64))
    o = P.combine_maps(a1, a2, 0.5, 0.25, 0.0)                   # (1.5, -1) before the norm
    rms = math.sqrt((1.5 ** 2 + 1.0) / 2)
    assert torch.allclose(o[1], torch.tensor([1.5, -1.0], dtype=F64) / rms * 0.75)
    assert torch.allclose(a1[0], v[0]) and torch.allclose(a2[0], v[0])    # the first sees itself


def test_plain_mix_weight():
    w = {"m.lq1": torch.tensor([1.0, 2.0]), "m.lk1": torch.tensor([0.5, 0.25]),
         "m.lq2": torch.tensor([1.0, 0.0]), "m.lk2": torch.tensor([0.1, 9.0])}
    lam = P.mix_weight({n: t.double() for n, t in w.items()}, "m.", 0.3)
    assert abs(float(lam) - (math.exp(1.0) - math.exp(0.1) + 0.3)) < 1e-7


def test_plain_clamped_feed_forward():
    """The gate is cut above only, the up projection on both sides and then shifted by one."""
    w = {"f.gate": torch.tensor([[1.0], [1.0], [1.0]], dtype=F64),
         "f.up": torch.tensor([[0.0], [5.0], [-5.0]], dtype=F64), "f.down": torch.eye(3, dtype=F64)}
    act = lambda g: g / (1 + math.exp(-1.702 * g))               # noqa: E731
    hi = P.clamped_mlp(torch.tensor([[9.0]], dtype=F64), w, "f.", 2.0)[0]
    assert torch.allclose(hi, torch.tensor([act(2.0), 3 * act(2.0), -act(2.0)], dtype=F64))
    lo = P.clamped_mlp(torch.tensor([[-9.0]], dtype=F64), w, "f.", 2.0)[0]
    assert torch.allclose(lo, torch.tensor([act(-9.0), -act(-9.0), 3 * act(-9.0)], dtype=F64))


def test_plain_router_counts_a_group_by_its_two_best():
    """Two groups of three.  Group 0 holds the single best expert, group 1 the better pair."""
    z = torch.tensor([[3.0, -4.0, -4.0, 1.0, 1.5, -9.0]], dtype=F64)
    w = {"r.router": torch.eye(6, dtype=F64)}
    ids, wts = P.route(z, w, "r.", {"top": 2, "groups": {"count": 2, "keep": 1}})
    assert sorted(ids[0].tolist()) == [3, 4]
    s = torch.sigmoid(z)[0]
    got = dict(zip(ids[0].tolist(), wts[0].tolist()))
    assert got[3] == float(s[3]) and got[4] == float(s[4])       # as they are
    ids, _ = P.route(z, w, "r.", {"top": 2})
    assert sorted(ids[0].tolist()) == [0, 4]
    ids, _ = P.route(z, w, "r.", {"top": 2, "groups": {"count": 6, "keep": 2}})
    assert sorted(ids[0].tolist()) == [0, 4]                     # groups of one expert
