"""Dense gated feed-forward: ``down( act(gate(x)) * up(x) )``, ``act`` silu (SwiGLU) or the
tanh form of gelu, or the clamped form ``min(g, c) sigmoid(a min(g, c)) (clamp(u, -c, c) + b)``
with three constants (``GatedMLPSpec.activation``; silu and the clamped form run in the products'
epilogues where those kernels apply, else the product and the activation kernel run).  With
``GatedMLPSpec.bias`` the three projections have biases: the first two are added (in float) where
the activation is applied, the last one rides on the add into the residual stream.

``silu(g) = g / (1 + exp(-g))`` (cuda/kernels/bf16_kernels.cu:461-477).  The
reference runs gate and up as two products (src/engine/batched_engine.ts:1243-1244);
here they are one product against the stacked weight ``[2 I, H]``, and the
activation kernel reads both halves of each output row.
"""
from __future__ import annotations

import os
from typing import Callable, List

import torch

from ..config.specs import GatedMLPSpec
from ..csrc import ops
from ..weights.loader import ParamSpec
from .base import (BuildEnv, DeferredLinear, FeedForward, ScaledRows, StackedOut, StepContext,
                   register_ffn, split_scaled)
from .linear import linear, pair_token_limit, swiglu_token_limit

# BINFER_B200_FUSE_SWIGLU=0: the stacked gate/up projection and the activation as two kernels
FUSE_SWIGLU = os.environ.get("BINFER_B200_FUSE_SWIGLU", "1") != "0"
# ... and only where its tiles (at least 16 outputs each) give work to this share of the SMs
FUSE_SWIGLU_FILL = 0.5


class GatedMLP(FeedForward, StackedOut):
    def __init__(self, spec: GatedMLPSpec, hidden_size: int, prefix: str, env: BuildEnv):
        if spec.activation not in ops.GATE_ACTIVATIONS:
            raise ValueError(f"activation {spec.activation!r} is not supported (supported: "
                             f"{sorted(ops.GATE_ACTIVATIONS)})")
        self.silu = spec.activation == "silu"
        self.fusable = spec.activation in ops.FUSED_ACTIVATIONS
        self._act = dict(activation=spec.activation, limit=spec.limit, slope=spec.slope,
                         up_offset=spec.up_offset)
        if spec.activation == "clamped" and not spec.limit > 0:
            raise ValueError("a clamped activation needs a positive limit")
        self.spec, self.hidden, self.prefix, self.env = spec, hidden_size, prefix, env
        self.inter = spec.intermediate_size
        self.out_cols = self.inter
        self.w_gate_up = self.w_out = None
        self.b_gate_up = self.out_bias = None   # float32, with GatedMLPSpec.bias
        self._swiglu_plan = None

    def param_specs(self) -> List[ParamSpec]:
        p = self.prefix
        gate, up, down = self.spec.names
        specs = [ParamSpec(p + gate, (self.inter, self.hidden)),
                 ParamSpec(p + up, (self.inter, self.hidden)),
                 ParamSpec(p + down, (self.hidden, self.inter))]
        if self.spec.bias:
            specs += [ParamSpec(p + n, (size,), init="around_zero", role="vector")
                      for n, size in zip(self.spec.bias_names,
                                         (self.inter, self.inter, self.hidden))]
        return specs

    def load(self, get: Callable[[ParamSpec], torch.Tensor]) -> None:
        g, u, d, *biases = self.param_specs()
        self.w_gate_up = torch.cat([get(g), get(u)], dim=0).contiguous()
        self.w_out = get(d)
        if biases:
            bg, bu, bd = (get(b) for b in biases)
            self.b_gate_up, self.out_bias = torch.cat([bg, bu]).contiguous(), bd

    accepts_scaled_rows = True

    def forward(self, x, ctx: StepContext) -> torch.Tensor:
        return self.forward_deferred(x, ctx).compute()

    def forward_deferred(self, x, ctx: StepContext) -> DeferredLinear:
        """Everything but the down projection (see ``GQAAttention.forward_deferred``)."""
        if isinstance(x, ScaledRows) and (self.inter % 8 or self.inter < 256 or not self.silu
                                          or self.spec.bias):
            x = x.dense()                  # the activation kernel takes the factor at other sizes only
        x, row_scale = split_scaled(x)
        h = torch.empty((x.shape[0], self.inter), dtype=x.dtype, device=x.device)
        self._inner(x, h, row_scale)
        return DeferredLinear(h, self.w_out, self.out_bias)

    def forward_inner(self, x, ctx: StepContext, view, out: torch.Tensor) -> bool:
        self._inner(x, out, None)
        return True

    def _inner(self, x, h, row_scale) -> None:
        """Gate, up and activation into ``h`` (which may be a column block of a wider buffer)."""
        if self._project_fused(x, h, row_scale):
            return
        gu = linear(x, self.w_gate_up)
        if self.silu and self.b_gate_up is None and h.is_contiguous():
            ops.silu_mul(gu, h, row_scale=row_scale)
        else:
            ops.gated_act_mul(gu, h, bias=self.b_gate_up, **self._act)

    def _project_fused(self, x, h, row_scale) -> bool:
        """Few token rows in bfloat16: the stacked projection with the activation in its
        epilogue, one CTA a tile of gate rows and the up rows of the same outputs.  False,
        having done nothing, where that kernel does not run."""
        if not FUSE_SWIGLU or not self.fusable or x.dtype != torch.bfloat16 or self.inter % 8:
            return False
        pair_from = pair_token_limit()
        if pair_from and x.shape[0] >= pair_from and row_scale is None:
            # many token rows: the product on pairs of SMs, the activation in its epilogue
            return ops.gemm_bf16_pair(x, self.w_gate_up, h, ops.error_word(x.device), gated=True,
                                      gate_bias=self.b_gate_up, **self._act)
        if x.shape[0] > swiglu_token_limit():
            return False
        if self._swiglu_plan is None:
            self._swiglu_plan = ops.gemm_swiglu_plan(self.inter, x.shape[1], x.device) or False
        plan = self._swiglu_plan
        if not plan or plan[1] < FUSE_SWIGLU_FILL * ops.num_sms(x.device):
            return False
        return ops.gemm_bf16_swiglu(x, self.w_gate_up, h, ops.error_word(x.device), plan[0],
                                    row_scale=row_scale, gate_bias=self.b_gate_up, **self._act)


register_ffn("gated_mlp", GatedMLP)
