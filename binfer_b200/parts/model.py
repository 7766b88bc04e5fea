"""The decoder: embedding, a schedule of layer executions, final norm, output head.

Built from a :class:`ModelSpec` alone.  The schedule is data: a list of
(layer, cache source) pairs that may run a layer twice or let an execution read
the pages of another one.  The reference hard-codes ``for layer in 0..L-1``
(src/engine/batched_engine.ts:1729-1731).

Output head (src/engine/batched_engine.ts:1733-1770): final norm, then logits
``y W^T`` with ``W = lm_head.weight`` or, when the embeddings are tied, the
embedding table (:1753-1755).  Only the rows whose logits are wanted go through
the norm and the head; logits are float32 (the reference's are bfloat16).
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..cache.manager import CacheManager, KVNeed, StateNeed
from ..config.specs import ModelSpec
from ..csrc import ops
from ..weights.loader import ParamSpec, TensorSource, check_names, place
from .base import (BuildEnv, DeferredLinear, EntryView, ResidualStream, StepContext, build_block,
                   build_norm)
from .linear import linear

# importing the modules registers the built-in parts
from . import attention as _attention  # noqa: F401
from . import attention_diff as _attention_diff  # noqa: F401
from . import attention_latent as _attention_latent  # noqa: F401
from . import attention_pooled as _attention_pooled  # noqa: F401
from . import delta_rule as _delta_rule  # noqa: F401
from . import mamba2 as _mamba2  # noqa: F401
from . import block as _block          # noqa: F401
from . import block_sublayer_norm as _block_sublayer_norm  # noqa: F401
from . import block_sandwich as _block_sandwich  # noqa: F401
from . import block_parallel as _block_parallel  # noqa: F401
from . import attention_conv_window as _attention_conv_window  # noqa: F401
from . import retention as _retention  # noqa: F401
from . import mixers_parallel as _mixers_parallel  # noqa: F401
from . import moe as _moe              # noqa: F401
from . import mlstm as _mlstm          # noqa: F401
from . import mlp as _mlp              # noqa: F401
from . import norms as _norms          # noqa: F401
from . import rope as _rope            # noqa: F401


class DecoderModel:
    def __init__(self, spec: ModelSpec, env: BuildEnv):
        self.spec, self.env = spec, env
        names = spec.names
        self.blocks = [build_block(ls, spec.hidden_size, names, i, env)
                       for i, ls in enumerate(spec.layers)]
        self.final_norm = build_norm(spec.final_norm, spec.hidden_size, names.final_norm, env)
        self.embed_spec = ParamSpec(names.embed, (spec.vocab_size, spec.hidden_size))
        self.head_spec = (None if spec.tie_word_embeddings
                          else ParamSpec(names.lm_head, (spec.vocab_size, spec.hidden_size)))
        self.embed: Optional[torch.Tensor] = None
        self.lm_head: Optional[torch.Tensor] = None
        # frequencies of the vectors that positions add to the embedding output, one per pair
        # of columns; double, so that the angle at a far position keeps its precision
        self.position_freqs: Optional[torch.Tensor] = None
        if spec.position_vectors is not None:
            i = torch.arange((spec.hidden_size + 1) // 2, dtype=torch.float64)
            self.position_freqs = torch.pow(
                torch.tensor(spec.position_vectors.base, dtype=torch.float64),
                -2.0 * i / spec.hidden_size).to(env.device)
        self.pass_spec = (None if spec.pass_table is None else
                          ParamSpec(spec.pass_table[0], (int(spec.pass_table[1]), spec.hidden_size),
                                    init="around_zero", role="vector"))
        self.pass_table: Optional[torch.Tensor] = None
        self.pass_proj_spec = (None if spec.pass_projection is None else
                               ParamSpec(spec.pass_projection,
                                         (spec.hidden_size, 2 * spec.hidden_size)))
        self.pass_proj: Optional[torch.Tensor] = None
        for e, entry in enumerate(spec.schedule):
            if entry.before is not None and entry.before.row is not None and not (
                    self.pass_spec is not None
                    and 0 <= entry.before.row < self.pass_spec.shape[0]):
                raise ValueError(f"schedule entry {e} adds row {entry.before.row} of a table "
                                 f"of pass vectors that the model lacks or that is shorter")
            if entry.before is not None and entry.before.project and (
                    self.pass_proj_spec is None or entry.before.embedding
                    or entry.before.row is not None):
                raise ValueError(f"schedule entry {e} projects the stream: the model needs a pass "
                                 f"projection, and nothing else is added there")
            if (entry.before is not None and (entry.before.embedding or entry.before.project)
                    and spec.position_vectors is not None):
                raise ValueError("the embedding output cannot be added again where positions "
                                 "add vectors to it")
            if not 0 <= entry.layer < len(self.blocks):
                raise ValueError(f"schedule entry {e} names layer {entry.layer}, "
                                 f"but there are {len(self.blocks)} layers")
            if entry.cache_from is not None:
                src = spec.schedule[entry.cache_from] if 0 <= entry.cache_from < e else None
                if src is None or src.cache_from is not None:
                    raise ValueError(f"schedule entry {e}: cache_from must name an earlier "
                                     f"entry that keeps a cache of its own")

    # ----------------------------------------------------------------- weights
    def param_specs(self) -> List[ParamSpec]:
        specs = [self.embed_spec]
        for b in self.blocks:
            specs += b.param_specs()
        specs += self.final_norm.param_specs()
        if self.pass_spec is not None:
            specs.append(self.pass_spec)
        if self.pass_proj_spec is not None:
            specs.append(self.pass_proj_spec)
        if self.head_spec is not None:
            specs.append(self.head_spec)
        return specs

    def load(self, source: TensorSource, allow_unexpected: bool = False) -> None:
        """Check every name and shape first (one error for all), then take the tensors.
        ``allow_unexpected``: tensors the model does not use are a warning, not an error."""
        optional = [self.spec.names.lm_head] if self.head_spec is None else []
        check_names(self.param_specs(), source.shapes, optional=optional, where=source.where,
                    allow_unexpected=allow_unexpected)

        def get(spec: ParamSpec) -> torch.Tensor:
            return place(source.get(spec.name), spec, self.env.dtype, self.env.device)

        self.embed = get(self.embed_spec)
        for b in self.blocks:
            b.load(get)
        self.final_norm.load(get)
        if self.pass_spec is not None:
            self.pass_table = get(self.pass_spec)
        if self.pass_proj_spec is not None:
            self.pass_proj = get(self.pass_proj_spec)
        self.lm_head = self.embed if self.head_spec is None else get(self.head_spec)

    def weight_bytes(self) -> int:
        """Bytes of every weight a step reads once (a tied table counts once per use)."""
        seen, total = set(), 0
        for obj in [self] + self.blocks + [self.final_norm] + \
                [p for b in self.blocks for p in (b.parts() if hasattr(b, "parts") else [])]:
            for v in vars(obj).values():
                # (by storage: a part's weight may be a column block of a stacked one)
                if isinstance(v, torch.Tensor) and v.untyped_storage().data_ptr() not in seen:
                    seen.add(v.untyped_storage().data_ptr())
                    total += v.untyped_storage().nbytes()
        return total

    # ------------------------------------------------------------------- cache
    def kv_needs(self) -> List[Optional[KVNeed]]:
        """Per schedule entry: the pages it keeps (None if it keeps none of its own)."""
        out: List[Optional[KVNeed]] = []
        for entry in self.spec.schedule:
            need = self.blocks[entry.layer].mixer.kv_need()
            out.append(need if entry.cache_from is None else None)
        # an execution that reads another's pages may look further back, or at pooled blocks
        # of another size: the pages are kept for the widest of them
        for entry in self.spec.schedule:
            if entry.cache_from is not None and out[entry.cache_from] is not None:
                need = self.blocks[entry.layer].mixer.kv_need()
                if need is not None and need != out[entry.cache_from]:
                    out[entry.cache_from] = out[entry.cache_from].merged(need)
        return out

    def state_needs(self) -> List[Optional[StateNeed]]:
        return [self.blocks[entry.layer].mixer.state_need() for entry in self.spec.schedule]

    def entry_views(self, cache: CacheManager) -> List[EntryView]:
        views: List[EntryView] = []
        for e, entry in enumerate(self.spec.schedule):
            src = e if entry.cache_from is None else entry.cache_from
            if cache.entry_location[src] is None:
                k = v = g = None
            else:
                k, v, g = cache.kv_view(src)
            views.append(EntryView(e, g, k, v, entry.cache_from is None, cache.state_storage[e],
                                   summaries=cache.summary_views(src)))
        return views

    # ----------------------------------------------------------------- forward
    def forward(self, ctx: StepContext, views: List[EntryView]) -> torch.Tensor:
        """Logits ``[R, vocab]`` (float32) at ``ctx.logit_rows``."""
        spec = self.spec
        resid = torch.empty((ctx.T, spec.hidden_size), dtype=torch.float32, device=self.env.device)
        ops.embed_gather(self.embed, ctx.token_ids, resid, spec.embedding_scale, ctx.err,
                         ctx.positions if self.position_freqs is not None else None,
                         self.position_freqs)
        stream = ResidualStream(resid)
        last = len(spec.schedule) - 1
        for e, entry in enumerate(spec.schedule):
            ctx.entry = e
            block = self.blocks[entry.layer]
            if entry.before is not None:
                self._open_pass(stream, ctx, entry.before, getattr(block, "first_norm", None))
            if getattr(block, "takes_successor", False):
                # a block may let its last product prepare the next block's first norm
                # (not where the stream changes in between: the start of a pass)
                nxt = (self.blocks[spec.schedule[e + 1].layer]
                       if e < last and spec.schedule[e + 1].before is None else None)
                block.forward(stream, ctx, views[e], nxt)
            else:
                block.forward(stream, ctx, views[e])
            if "layer_outputs" in ctx.scratch:
                # for tests and debugging: the stream after every layer run, everything folded in
                stream.flush()
                ctx.scratch["layer_outputs"].append(stream.x.clone())
        R = ctx.logit_rows.shape[0]
        if R == 0:
            stream.flush()
            return torch.empty((0, spec.vocab_size), dtype=torch.float32, device=self.env.device)
        y = stream.norm_input(self.final_norm, rows=ctx.logit_rows, n_rows=R)
        logits = linear(y, self.lm_head, out_dtype=torch.float32)
        if spec.logit_scale != 1.0:
            logits.mul_(spec.logit_scale)
        return logits


    def _open_pass(self, stream: ResidualStream, ctx: StepContext, before, norm=None) -> None:
        """Fold the pending sublayer output into the stream together with what a pass starts
        with: the embedding output again (gathered from the table anew, in float) and a row
        of the pass table; or replace the stream by the pass projection of itself and the
        embedding output.  ``norm``: the norm that reads the stream next, if the block says so."""
        if before.project:
            pair = torch.empty((ctx.T, 2 * self.spec.hidden_size), dtype=self.env.dtype,
                               device=self.env.device)
            ops.stream_pair(stream.x, stream.pending, stream.pending2, stream.pending_bias,
                            self.embed, ctx.token_ids, self.spec.embedding_scale, pair, ctx.err)
            stream.replace_linear(DeferredLinear(pair, self.pass_proj), norm)
            return
        if not before.embedding and before.row is None:
            return
        if stream.pending2 is not None or stream.pending_bias is not None:
            stream.flush()
        delta, stream.pending = stream.pending, None
        stream.ready = stream.ready_for = stream.reading = None
        ops.stream_inject(stream.x, delta, self.embed if before.embedding else None,
                          ctx.token_ids, self.spec.embedding_scale,
                          self.pass_table[before.row] if before.row is not None else None, ctx.err)


def param_specs_for(spec: ModelSpec) -> List[ParamSpec]:
    """Names, shapes and roles of every tensor a checkpoint of ``spec`` must hold."""
    env = BuildEnv(torch.float32, torch.device("cpu"))
    return DecoderModel(spec, env).param_specs()


def build_model(spec: ModelSpec, env: BuildEnv, source: TensorSource,
                allow_unexpected: bool = False) -> DecoderModel:
    model = DecoderModel(spec, env)
    model.load(source, allow_unexpected=allow_unexpected)
    return model
