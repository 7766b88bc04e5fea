"""Typed configuration of the Nazorax decoder, read from its config.json keys.

A Nazorax layer has one norm and both sublayers read its output, ``h = norm1(x);  x += mixer(h)
+ ff(h)`` (``mlp: null``: no feed-forward).  The norm takes no statistic of the row: ``tanh(alpha
x) * w + b`` with one number alpha.  Each layer names one of two mixers:

* ``attention``: grouped softmax attention over a sliding window, q, k and v with biases,
  rotary positions in halves on the first sizes of a head;
* ``latent_attention``: softmax attention whose keys and values are expanded from one cached
  latent vector per token, with one rotated key part that all heads share (rotary positions in
  halves, optionally stretched by pair index, ``rot.scaling``) and a learned logit per head in the
  softmax's denominator.

The feed-forward is dense (``silu``, every projection with a bias) or a mixture of experts of
the clamped form (no biases), whose router weighs the chosen experts by the softmax over their
logits alone, with a shared expert that runs for every token.

``loop`` walks the layers ``start .. stop - 1`` ``times`` times in a row with the same weights;
every pass keeps a cache of its own.  Before every pass the stream x becomes ``W [x; x0]``, W the
tensor ``loop.in`` and x0 the embedding output.  The model ends in its norm (``final.norm``) and an
output head.

Keys: ``architecture``, ``vocab``, ``width``, ``norm.eps``, ``layers``, ``loop.{start, stop,
times}``; of a layer ``type``, ``mixer``, ``mlp``; of attention ``heads, kv_heads, dim, vdim, scale,
mask.size, rot.{base, dims}``; of latent attention ``heads, dim, rot_dim, vdim, kv_rank, scale,
rot.{base, dims, scaling.{factor, original, fast, slow}}``; of a dense feed-forward ``kind, ff``;
of a mixture ``kind, router.{experts, top}, expert.{ff, limit}, shared.{ff, limit}``.  Tensors:
``embed``, ``head``, ``final.norm``, ``loop.in`` and ``l<i>.{norm1, mix.*, mlp.*}``; a norm's name
with ``.alpha`` and ``.b``, a projection's with ``.b``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .ketopel import _need, _positive, _rope
from .specs import (ConfigError, ConvWindowAttentionSpec, GatedMLPSpec, LatentAttentionSpec,
                    LayerSpec, ModelSpec, MoESpec, NameLayout, NormSpec, PassStart,
                    ScheduleEntry)

PASS_PROJECTION_NAME = "loop.in"
BIAS_SUFFIX = ".b"
ALPHA_SUFFIX = ".alpha"
EXPERT_SLOPE = 1.702         # experts: g sigmoid(slope g) (u + offset)
EXPERT_UP_OFFSET = 1.0
_MLP_NAMES = ("gate", "up", "down")


def _limit(d: Dict[str, Any], where: str) -> float:
    v = float(_need(d, "limit", where))
    if not v > 0:
        raise ConfigError(f"{where}limit must be positive, got {v}")
    return v


@dataclass(frozen=True)
class NazoraxConfig:
    raw: Dict[str, Any]
    vocab_size: int
    hidden_size: int
    norm_eps: float
    layers: Tuple[LayerSpec, ...]
    loop: Optional[Tuple[int, int, int]]        # (start, stop, times)
    architectures: Tuple[str, ...] = ("Nazorax",)

    # ------------------------------------------------------------------ parse
    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "NazoraxConfig":
        width = _positive(_need(raw, "width", ""), "width")
        vocab = _positive(_need(raw, "vocab", ""), "vocab")
        eps = float(_need(_need(raw, "norm", ""), "eps", "norm."))
        if not eps > 0:
            raise ConfigError(f"norm.eps must be positive, got {eps}")
        entries = _need(raw, "layers", "")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("layers must be a non-empty list")
        parsers = {"attention": cls._attention, "latent_attention": cls._latent}
        layers: List[LayerSpec] = []
        for i, entry in enumerate(entries):
            where = f"layers[{i}]."
            kind = _need(entry, "type", where)
            if kind not in parsers:
                raise ConfigError(f"{where}type {kind!r} is not supported (supported: "
                                  f"{sorted(parsers)})")
            mixer = parsers[kind](_need(entry, "mixer", where), eps, where + "mixer.")
            layers.append(LayerSpec(mixer=mixer, ffn=cls._mlp(entry.get("mlp"), where + "mlp."),
                                    norm=cls._norm(eps), block="parallel"))
        loop = None
        lp = raw.get("loop")
        if lp:
            start, stop = int(_need(lp, "start", "loop.")), int(_need(lp, "stop", "loop."))
            times = _positive(_need(lp, "times", "loop."), "loop.times")
            if not 0 <= start < stop <= len(layers):
                raise ConfigError(f"loop: start {start} and stop {stop} must name a run of the "
                                  f"{len(layers)} layers")
            loop = (start, stop, times)
        return cls(raw=copy.deepcopy(raw), vocab_size=vocab, hidden_size=width, norm_eps=eps,
                   layers=tuple(layers), loop=loop,
                   architectures=(str(raw.get("architecture", "Nazorax")),))

    @staticmethod
    def _norm(eps: float) -> NormSpec:
        return NormSpec(kind="tanh_norm", eps=eps, bias_suffix=BIAS_SUFFIX,
                        alpha_suffix=ALPHA_SUFFIX)

    @staticmethod
    def _attention(mx: Dict[str, Any], eps: float, where: str) -> ConvWindowAttentionSpec:
        heads = _positive(_need(mx, "heads", where), where + "heads")
        kv_heads = _positive(mx.get("kv_heads") or heads, where + "kv_heads")
        if heads % kv_heads:
            raise ConfigError(f"{where}heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
        dim = _positive(_need(mx, "dim", where), where + "dim")
        window = (mx.get("mask") or {}).get("size")
        if window is not None:
            window = _positive(window, where + "mask.size")
        return ConvWindowAttentionSpec(
            num_heads=heads, num_kv_heads=kv_heads, head_dim=dim,
            value_dim=_positive(mx.get("vdim") or dim, where + "vdim"), conv_taps=0,
            position=_rope(mx.get("rot"), dim, where + "rot."), unit_norm=False, norm_eps=eps,
            scale=float(_need(mx, "scale", where)), window=window, keep_first=0, sinks=False, proj_bias=True,
            bias_suffix=BIAS_SUFFIX)

    @staticmethod
    def _latent(mx: Dict[str, Any], eps: float, where: str) -> LatentAttentionSpec:
        rot_dim = _positive(_need(mx, "rot_dim", where), where + "rot_dim")
        return LatentAttentionSpec(
            num_heads=_positive(_need(mx, "heads", where), where + "heads"),
            head_dim=_positive(_need(mx, "dim", where), where + "dim"), rot_dim=rot_dim,
            value_dim=_positive(_need(mx, "vdim", where), where + "vdim"),
            kv_rank=_positive(_need(mx, "kv_rank", where), where + "kv_rank"),
            scale=float(_need(mx, "scale", where)), norm_eps=eps,
            position=_rope(_need(mx, "rot", where), rot_dim, where + "rot.", "half", rot_dim),
            head_gate=False, sinks=True)

    @staticmethod
    def _mlp(mlp: Optional[Dict[str, Any]], where: str):
        if mlp is None:
            return None
        kind = _need(mlp, "kind", where)
        if kind == "dense":
            return GatedMLPSpec(
                intermediate_size=_positive(_need(mlp, "ff", where), where + "ff"),
                activation="silu", bias=True, names=_MLP_NAMES,
                bias_names=tuple(n + BIAS_SUFFIX for n in _MLP_NAMES))
        if kind != "moe":
            raise ConfigError(f"{where}kind {kind!r} is not supported (supported: 'dense', 'moe')")
        router = _need(mlp, "router", where)
        experts = _positive(_need(router, "experts", where + "router."), where + "router.experts")
        top = _positive(_need(router, "top", where + "router."), where + "router.top")
        if top > experts:
            raise ConfigError(f"{where}router.top ({top}) exceeds router.experts ({experts})")
        expert = _need(mlp, "expert", where)
        shared = mlp.get("shared")
        w = where + "shared."
        return MoESpec(
            num_experts=experts, top=top,
            expert_size=_positive(_need(expert, "ff", where + "expert."), where + "expert.ff"),
            shared_size=_positive(_need(shared, "ff", w), w + "ff") if shared else 0,
            shared_gate=False, activation="clamped", limit=_limit(expert, where + "expert."),
            shared_limit=_limit(shared, w) if shared else 0.0, slope=EXPERT_SLOPE,
            up_offset=EXPERT_UP_OFFSET, names=_MLP_NAMES)

    # ------------------------------------------------------------- derivation
    def schedule(self) -> Tuple[ScheduleEntry, ...]:
        """One entry per layer run; a looped run of layers repeats, and the stream is projected
        before the first entry of every pass."""
        n = len(self.layers)
        if self.loop is None:
            return tuple(ScheduleEntry(i) for i in range(n))
        start, stop, times = self.loop
        out = [ScheduleEntry(i) for i in range(start)]
        for _ in range(times):
            for i in range(start, stop):
                out.append(ScheduleEntry(i, None, PassStart(project=True) if i == start else None))
        return tuple(out + [ScheduleEntry(i) for i in range(stop, n)])

    def to_spec(self) -> ModelSpec:
        names = NameLayout(embed="embed", layer_prefix="l{i}.", input_norm="norm1",
                           post_mixer_norm="norm2", mixer="mix", ffn="mlp",
                           final_norm="final.norm", lm_head="head", norm_suffix="")
        return ModelSpec(
            architecture=self.architectures[0], hidden_size=self.hidden_size,
            vocab_size=self.vocab_size, layers=self.layers, schedule=self.schedule(),
            final_norm=self._norm(self.norm_eps), tie_word_embeddings=False,
            max_position_embeddings=1 << 30, eos_token_ids=(), bos_token_id=None,
            pad_token_id=None, names=names,
            pass_projection=PASS_PROJECTION_NAME if self.loop is not None else None)

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
