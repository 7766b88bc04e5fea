"""Arrangement of a layer's parts with one norm that both sublayers read.

``h = norm(x);  x += mixer(h) + ffn(h)`` (a layer may have no feed-forward).  Where both parts
can hand over what lies in front of their last product (``StackedOut``), the two products are
one, against both weights side by side: the sum of the sublayers is formed in its accumulation,
and for few token rows its epilogue adds it into the stream and makes the next norm's output
(``ResidualStream.add_linear``).  Otherwise the mixer's output is left pending on the residual
stream and the feed-forward's rides beside it as a second pending add; the next norm (this
arrangement's, or the model's final one) folds both into the float stream in the pass that norms
it.
"""
from __future__ import annotations

import os
from typing import List, Optional

import torch

from ..config.specs import LayerSpec, NameLayout
from .base import (BuildEnv, DeferredLinear, EntryView, Part, ResidualStream, StackedOut,
                   StepContext, build_ffn, build_mixer, build_norm, register_block)
from .linear import linear

# BINFER_B200_STACK_OUT=0: the two sublayers' last products apart
STACK_OUT = os.environ.get("BINFER_B200_STACK_OUT", "1") != "0"


class ParallelBlock(Part):
    takes_successor = True      # forward(stream, ctx, view, successor): see DecoderModel.forward

    def __init__(self, spec: LayerSpec, hidden_size: int, names: NameLayout, index: int,
                 env: BuildEnv):
        p = names.layer_prefix.format(i=index)
        self.index, self.env = index, env
        self.norm = build_norm(spec.norm, hidden_size,
                               f"{p}{names.norm('input')}{names.norm_suffix}", env)
        self.mixer = build_mixer(spec.mixer, hidden_size, f"{p}{names.mixer}.", env)
        self.ffn = (build_ffn(spec.ffn, hidden_size, f"{p}{names.ffn}.", env)
                    if spec.ffn is not None else None)
        self.stacked = (STACK_OUT and isinstance(self.mixer, StackedOut)
                        and (self.ffn is None or isinstance(self.ffn, StackedOut)))
        self.w_out: Optional[torch.Tensor] = None

    def parts(self) -> List[Part]:
        return [p for p in (self.norm, self.mixer, self.ffn) if p is not None]

    @property
    def first_norm(self):
        """The norm that reads the stream first."""
        return self.norm

    def param_specs(self):
        return [s for part in self.parts() for s in part.param_specs()]

    def load(self, get) -> None:
        for part in self.parts():
            part.load(get)
        if self.stacked and self.ffn is not None:
            a, b = self.mixer, self.ffn
            self.w_out = torch.cat([a.w_out, b.w_out], dim=1).contiguous()
            # (for steps in which a part has a way of its own)
            a.w_out, b.w_out = self.w_out[:, :a.out_cols], self.w_out[:, a.out_cols:]

    def forward(self, stream: ResidualStream, ctx: StepContext, view: EntryView,
                successor: Optional[Part] = None) -> None:
        """``successor``: the block that runs next on this stream, if any; its norm can then be
        prepared by this block's last product."""
        h = stream.norm_input(self.norm)
        if self.stacked:
            self._forward_stacked(h, stream, ctx, view, getattr(successor, "first_norm", None))
            return
        y = self.mixer.forward(h, ctx, view)
        if self.ffn is None:
            stream.add(y)
            return
        deferred = getattr(self.ffn, "forward_deferred", None)
        if deferred is None:
            stream.add_pair(y, self.ffn.forward(h, ctx))
        else:
            d = deferred(h, ctx)        # (its bias rides on the adds)
            stream.add_pair(y, linear(d.x, d.w), d.bias)

    def _forward_stacked(self, h, stream: ResidualStream, ctx: StepContext, view: EntryView,
                         next_norm) -> None:
        m, f, n = self.mixer, self.ffn, self.mixer.out_cols
        acts = torch.empty((h.shape[0], n + (f.out_cols if f is not None else 0)), dtype=h.dtype,
                           device=h.device)
        m.forward_inner(h, ctx, view, acts[:, :n])
        if f is None:
            stream.add_linear(DeferredLinear(acts, m.w_out, m.out_bias), next_norm)
        elif f.forward_inner(h, ctx, None, acts[:, n:]):
            bias = m.out_bias if f.out_bias is None else f.out_bias
            if m.out_bias is not None and f.out_bias is not None:
                bias = m.out_bias + f.out_bias
            stream.add_linear(DeferredLinear(acts, self.w_out, bias), next_norm)
        else:
            y = f.forward(h, ctx)
            stream.add(y)
            stream.add_linear(DeferredLinear(acts[:, :n], m.w_out, m.out_bias), next_norm)


register_block("parallel", ParallelBlock)
