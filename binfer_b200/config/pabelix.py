"""Typed configuration of the Pabelix decoder, read from its config.json keys.

A Pabelix layer has a norm before and after each sublayer, ``x += norm1b(mixer(norm1(x)));
x += norm2b(ff(norm2(x)))`` (``mlp: null``: the first half only), with RMS norms whose stored
weight is the deviation from one (the model's last norm too).  The embedding output is
``embed[token]`` plus a sinusoidal vector of the position; there is no rotation.  The one mixer,
``attention``, is differential attention: each head is the normed difference of two softmax
maps over the same values, with a query temperature that grows with the logarithm of the
position and a gate on the output.  A layer with ``kv_from`` reads an earlier layer's keys and
values.  The feed-forward is dense, with a clamped gate and a clamped, shifted up projection,
or a mixture of gated experts (``silu``) whose router scores by sigmoids, chooses inside the
groups with the largest sum of two scores, and weighs by the scores as they are.  The output
head is the embedding table.

Keys: ``architecture``, ``vocab``, ``width``, ``norm.eps``, ``layers``; of a layer ``type``,
``mixer.{heads, kv_heads, dim, vdim, scale, diff, q_temp.{coef, every}, kv_from}``, ``mlp.{kind,
ff, limit}`` or ``mlp.{kind, expert.ff, router.{experts, top, groups.{count, keep}}}``.
Tensors: ``embed``, ``final.norm`` and ``l<i>.{norm1, norm1b, norm2, norm2b, mix.*, mlp.{gate,
up, down}}`` or ``l<i>.mlp.{e<j>.{gate, up, down}, router}``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .specs import (ConfigError, DifferentialAttentionSpec, GatedMLPSpec, LayerSpec, ModelSpec,
                    MoESpec, NameLayout, NormSpec, PositionVectorSpec, ScheduleEntry)

# constants of the design, in no config.json
NORM_WEIGHT_OFFSET = 1.0         # the norms' stored weights are deviations from it
POSITION_BASE = 10000.0
GATE_SLOPE, UP_OFFSET = 1.702, 1.0
GROUP_TOP = 2                    # a group of experts counts by its two largest scores
_MLP_NAMES = ("gate", "up", "down")


def _need(d: Dict[str, Any], key: str, where: str) -> Any:
    if not isinstance(d, dict) or key not in d or d[key] is None:
        raise ConfigError(f"Missing required config key: {where}{key}")
    return d[key]


def _positive(v: Any, what: str) -> int:
    if isinstance(v, bool) or int(v) != v or int(v) <= 0:
        raise ConfigError(f"{what} must be a positive integer, got {v!r}")
    return int(v)


@dataclass(frozen=True)
class PabelixConfig:
    raw: Dict[str, Any]
    vocab_size: int
    hidden_size: int
    norm_eps: float
    layers: Tuple[LayerSpec, ...]
    # per layer: the layer whose keys and values it reads (None: its own)
    cache_from: Tuple[Optional[int], ...]
    architectures: Tuple[str, ...] = ("Pabelix",)

    # ------------------------------------------------------------------ parse
    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "PabelixConfig":
        width = _positive(_need(raw, "width", ""), "width")
        vocab = _positive(_need(raw, "vocab", ""), "vocab")
        eps = float(_need(_need(raw, "norm", ""), "eps", "norm."))
        if not eps > 0:
            raise ConfigError(f"norm.eps must be positive, got {eps}")
        entries = _need(raw, "layers", "")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("layers must be a non-empty list")
        norm = NormSpec(kind="rmsnorm", eps=eps, offset=NORM_WEIGHT_OFFSET)
        layers: List[LayerSpec] = []
        cache_from: List[Optional[int]] = []
        for i, entry in enumerate(entries):
            where = f"layers[{i}]."
            kind = _need(entry, "type", where)
            if kind != "attention":
                raise ConfigError(f"{where}type {kind!r} is not supported (supported: "
                                  f"'attention')")
            mixer, src = cls._attention(_need(entry, "mixer", where), eps, where + "mixer.")
            layers.append(LayerSpec(mixer=mixer, ffn=cls._mlp(entry.get("mlp"), where + "mlp."),
                                    norm=norm, block="sandwich"))
            cache_from.append(src)
        for i, src in enumerate(cache_from):
            if src is None:
                continue
            if not 0 <= src < i or cache_from[src] is not None:
                raise ConfigError(f"layers[{i}].mixer.kv_from must name an earlier layer with "
                                  f"keys and values of its own, got {src}")
            a, b = layers[i].mixer, layers[src].mixer
            if (a.num_kv_heads, a.head_dim, a.value_dim) != (b.num_kv_heads, b.head_dim,
                                                             b.value_dim):
                raise ConfigError(f"layers[{i}] reads the keys and values of layers[{src}], "
                                  f"whose head count or sizes differ")
        return cls(raw=copy.deepcopy(raw), vocab_size=vocab, hidden_size=width, norm_eps=eps,
                   layers=tuple(layers), cache_from=tuple(cache_from),
                   architectures=(str(raw.get("architecture", "Pabelix")),))

    @staticmethod
    def _attention(mx: Dict[str, Any], eps: float, where: str):
        heads = _positive(_need(mx, "heads", where), where + "heads")
        kv_heads = _positive(mx.get("kv_heads") or heads, where + "kv_heads")
        if heads % kv_heads:
            raise ConfigError(f"{where}heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
        dim = _positive(_need(mx, "dim", where), where + "dim")
        temp = mx.get("q_temp") or {}
        coef, every = 0.0, 1
        if temp:
            coef = float(_need(temp, "coef", where + "q_temp."))
            every = _positive(_need(temp, "every", where + "q_temp."), where + "q_temp.every")
        src = mx.get("kv_from")
        if src is not None and (isinstance(src, bool) or int(src) != src):
            raise ConfigError(f"{where}kv_from must be a layer's number, got {src!r}")
        spec = DifferentialAttentionSpec(
            num_heads=heads, num_kv_heads=kv_heads, head_dim=dim,
            value_dim=_positive(mx.get("vdim") or dim, where + "vdim"),
            scale=float(_need(mx, "scale", where)), diff=float(_need(mx, "diff", where)),
            norm_eps=eps, temp_coef=coef, temp_every=every, output_gate=True,
            own_cache=src is None)
        return spec, (None if src is None else int(src))

    @staticmethod
    def _mlp(mlp: Optional[Dict[str, Any]], where: str):
        if mlp is None:
            return None
        kind = _need(mlp, "kind", where)
        if kind == "dense":
            limit = float(_need(mlp, "limit", where))
            if not limit > 0:
                raise ConfigError(f"{where}limit must be positive, got {limit}")
            return GatedMLPSpec(
                intermediate_size=_positive(_need(mlp, "ff", where), where + "ff"),
                activation="clamped", limit=limit, slope=GATE_SLOPE, up_offset=UP_OFFSET,
                names=_MLP_NAMES)
        if kind != "moe":
            raise ConfigError(f"{where}kind {kind!r} is not supported (supported: 'dense', 'moe')")
        router = _need(mlp, "router", where)
        w = where + "router."
        experts = _positive(_need(router, "experts", w), w + "experts")
        top = _positive(_need(router, "top", w), w + "top")
        groups = router.get("groups") or {}
        count = _positive(groups.get("count") or 1, w + "groups.count")
        keep = _positive(groups.get("keep") or count, w + "groups.keep")
        if experts % count or keep > count:
            raise ConfigError(f"{w}groups: {count} groups must divide the {experts} experts, and "
                              f"keep ({keep}) not exceed them")
        if top > keep * (experts // count):
            raise ConfigError(f"{w}top ({top}) exceeds what {keep} groups hold")
        return MoESpec(
            num_experts=experts, top=top,
            expert_size=_positive(_need(_need(mlp, "expert", where), "ff", where + "expert."),
                                  where + "expert.ff"),
            activation="silu", scoring="sigmoid", normalize=False, groups=count, groups_keep=keep,
            group_top=GROUP_TOP)

    # ------------------------------------------------------------- derivation
    def to_spec(self) -> ModelSpec:
        names = NameLayout(embed="embed", layer_prefix="l{i}.", input_norm="norm1",
                           post_mixer_norm="norm2", mixer="mix", ffn="mlp",
                           final_norm="final.norm", lm_head="head", norm_suffix="",
                           more_norms=(("mixer_out", "norm1b"), ("ffn_out", "norm2b")))
        return ModelSpec(
            architecture=self.architectures[0], hidden_size=self.hidden_size,
            vocab_size=self.vocab_size, layers=self.layers,
            schedule=tuple(ScheduleEntry(i, src) for i, src in enumerate(self.cache_from)),
            final_norm=NormSpec(kind="rmsnorm", eps=self.norm_eps, offset=NORM_WEIGHT_OFFSET),
            tie_word_embeddings=True, max_position_embeddings=1 << 30, eos_token_ids=(),
            bos_token_id=None, pad_token_id=None, names=names,
            position_vectors=PositionVectorSpec(base=POSITION_BASE))

    def to_dict(self) -> Dict[str, Any]:
        """The config.json that :meth:`from_dict` reads back to this object."""
        return copy.deepcopy(self.raw)

    # ---------------------------------------------------------------- memory
    def num_parameters(self) -> int:
        from ..parts.model import param_specs_for
        total = 0
        for s in param_specs_for(self.to_spec()):
            n = 1
            for d in s.shape:
                n *= d
            total += n
        return total
