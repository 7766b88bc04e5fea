"""Arrangement of a layer's parts with a norm before and a norm after each sublayer.

``x += norm_out(mixer(norm_in(x)))`` and, where the layer has a feed-forward, the same around it
with two norms of its own.  The norm of a sublayer's output, the add into the float stream and
the norm that reads the new stream next (this layer's second, or the following layer's first)
are one kernel (``Norm.add_normed``); only the first norm of a model is a launch of its own.
"""
from __future__ import annotations

from typing import List, Optional

from ..config.specs import LayerSpec, NameLayout
from .base import (BuildEnv, EntryView, Part, ResidualStream, ScaledRows, StepContext, build_ffn,
                   build_mixer, build_norm, register_block)


class SandwichBlock(Part):
    takes_successor = True      # forward(stream, ctx, view, successor): see DecoderModel.forward

    def __init__(self, spec: LayerSpec, hidden_size: int, names: NameLayout, index: int,
                 env: BuildEnv):
        p = names.layer_prefix.format(i=index)

        def norm(role: str):
            return build_norm(spec.norm, hidden_size, f"{p}{names.norm(role)}{names.norm_suffix}",
                              env)

        self.index = index
        self.input_norm = norm("input")
        self.mixer = build_mixer(spec.mixer, hidden_size, f"{p}{names.mixer}.", env)
        self.mixer_out_norm = norm("mixer_out")
        self.ffn_in_norm = self.ffn = self.ffn_out_norm = None
        if spec.ffn is not None:
            self.ffn_in_norm = norm("post_mixer")
            self.ffn = build_ffn(spec.ffn, hidden_size, f"{p}{names.ffn}.", env)
            self.ffn_out_norm = norm("ffn_out")

    def parts(self) -> List[Part]:
        return [part for part in (self.input_norm, self.mixer, self.mixer_out_norm,
                                  self.ffn_in_norm, self.ffn, self.ffn_out_norm)
                if part is not None]

    def param_specs(self):
        return [s for part in self.parts() for s in part.param_specs()]

    def load(self, get) -> None:
        for part in self.parts():
            part.load(get)

    def forward(self, stream: ResidualStream, ctx: StepContext, view: EntryView,
                successor: Optional[Part] = None) -> None:
        after = successor.input_norm if isinstance(successor, SandwichBlock) else None
        y = self.mixer.forward(self._dense(self.input_norm.forward(stream)), ctx, view)
        if self.ffn is None:
            self.mixer_out_norm.add_normed(stream, y, after)
            return
        self.mixer_out_norm.add_normed(stream, y, self.ffn_in_norm)
        y = self.ffn.forward(self._dense(self.ffn_in_norm.forward(stream)), ctx)
        self.ffn_out_norm.add_normed(stream, y, after)

    @staticmethod
    def _dense(h):
        return h.dense() if isinstance(h, ScaledRows) else h


register_block("sandwich", SandwichBlock)
