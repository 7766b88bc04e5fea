"""Differential attention over the paged cache, as a mixer part.

Each query and key head holds two vectors side by side, one per map; both maps are causal
softmax attentions over the same values.  A head's result is the first map's output minus a
learned number (one for the layer) times the second's, divided by its root mean square, times a
constant, times the sigmoid of a projection of the mixer's input, element by element; the
output projection follows.  Queries may count more the farther their position (a factor that
grows with the logarithm of the position in steps).

One product yields q, k, v and the gate of a token side by side.  A kernel stores k (both maps'
keys of a head as one cache row) and v into the pages; everything between that and the output
projection is the attention kernel: it reads q and the gate from the product's rows, takes the
query's factor into the scores, and leaves the gated heads.  A layer that reads another layer's
keys and values has neither in its product and skips the store.

Which kernel: float32, and sizes that the tensor-core kernels do not take, run one warp per
(token, head), whose sums have one fixed order per position.  bfloat16: rows that bring a
single token and prompt portions go to kernels of their own, as in ``attention.GQAAttention``.
"""
from __future__ import annotations

import math
import os
from typing import Callable, List, Optional

import torch

from ..cache.manager import KVNeed
from ..config.specs import DifferentialAttentionSpec
from ..csrc import ops
from ..weights.loader import ParamSpec
from .base import BuildEnv, EntryView, Mixer, StepContext, register_mixer
from .linear import linear

# BINFER_B200_DIFF_TENSOR_CORES=0: the one-warp-per-row kernel also in bfloat16
TENSOR_CORES = os.environ.get("BINFER_B200_DIFF_TENSOR_CORES", "1") != "0"


class DifferentialAttention(Mixer):
    def __init__(self, spec: DifferentialAttentionSpec, hidden_size: int, prefix: str,
                 env: BuildEnv):
        s = spec
        if s.num_heads % s.num_kv_heads:
            raise ValueError("num_heads must be a multiple of num_kv_heads")
        if not 0 < s.head_dim <= ops.DIFF_MAX_DIM or not 0 < s.value_dim <= ops.DIFF_MAX_DIM:
            raise ValueError(f"differential attention: sizes {s.head_dim}, {s.value_dim} are not "
                             f"supported (at most {ops.DIFF_MAX_DIM})")
        if s.temp_every < 1:
            raise ValueError("differential attention: temp_every must be positive")
        self.spec, self.hidden, self.prefix, self.env = spec, hidden_size, prefix, env
        self.H, self.G, self.d, self.dv = s.num_heads, s.num_kv_heads, s.head_dim, s.value_dim
        self.q_size, self.k_size = self.H * 2 * self.d, self.G * 2 * self.d
        self.v_size, self.o_size = self.G * self.dv, self.H * self.dv
        # columns of the stacked product: q, then (own cache) k and v, then the gate
        self.k_off = self.q_size
        self.v_off = self.k_off + (self.k_size if s.own_cache else 0)
        self.gate_off = self.v_off + (self.v_size if s.own_cache else 0)
        self.names = dict(s.names)
        self.w_proj = self.w_o = None
        self.lam = 0.0

    # ----------------------------------------------------------------- weights
    def _spec(self, role: str) -> ParamSpec:
        n = self.prefix + self.names[role]
        if role in ("lq1", "lk1", "lq2", "lk2"):
            return ParamSpec(n, (self.d,), init="around_zero", role="vector")
        return ParamSpec(n, {"q": (self.q_size, self.hidden), "k": (self.k_size, self.hidden),
                             "v": (self.v_size, self.hidden), "g": (self.o_size, self.hidden),
                             "o": (self.hidden, self.o_size)}[role])

    def _proj_roles(self) -> List[str]:
        s = self.spec
        return ["q"] + (["k", "v"] if s.own_cache else []) + (["g"] if s.output_gate else [])

    def param_specs(self) -> List[ParamSpec]:
        return [self._spec(r) for r in self._proj_roles() + ["o", "lq1", "lk1", "lq2", "lk2"]]

    def load(self, get: Callable[[ParamSpec], torch.Tensor]) -> None:
        g = lambda role: get(self._spec(role))          # noqa: E731
        self.w_proj = torch.cat([g(r) for r in self._proj_roles()], dim=0).contiguous()
        self.w_o = g("o")
        dot = lambda a, b: float((g(a).double() * g(b).double()).sum())     # noqa: E731
        self.lam = math.exp(dot("lq1", "lk1")) - math.exp(dot("lq2", "lk2")) + self.spec.diff

    # ------------------------------------------------------------------- cache
    def kv_need(self) -> Optional[KVNeed]:
        # a cached key head is the keys of both maps side by side
        return KVNeed(self.G, 2 * self.d, None, None if self.dv == 2 * self.d else self.dv)

    # ----------------------------------------------------------------- forward
    def forward(self, x: torch.Tensor, ctx: StepContext, view: EntryView) -> torch.Tensor:
        s, T = self.spec, x.shape[0]
        if view.writes_cache != s.own_cache:
            raise ValueError("a layer with key and value tensors keeps a cache of its own, "
                             "one without reads another's")
        proj = linear(x, self.w_proj)
        if s.own_cache:
            ops.kv_store(proj, self.k_off, self.v_off, ctx.slots[view.group], view.k_cache,
                         view.v_cache, ctx.err)
        out = torch.empty((T, self.o_size), dtype=x.dtype, device=x.device)
        gate = proj[:, self.gate_off:self.gate_off + self.o_size] if s.output_gate else None
        self.attend(proj[:, :self.q_size], gate, out, ctx, view)
        return linear(out, self.w_o)

    def attend(self, q: torch.Tensor, gate: Optional[torch.Tensor], out: torch.Tensor,
               ctx: StepContext, view: EntryView) -> None:
        s = self.spec
        dc = ops.DiffCombine(self.lam, s.norm_eps, 1.0 - s.diff, gate, s.temp_coef, s.temp_every)
        tables = ctx.block_tables[view.group]
        if not TENSOR_CORES or not ops.diff_attention_takes(q.dtype, self.d, self.dv,
                                                            s.softmax_scale, s.temp_coef):
            ops.diff_attention_generic(q, view.k_cache, view.v_cache, ctx.seq_of_token,
                                       ctx.positions, tables, out, self.H, s.softmax_scale, dc,
                                       ctx.err)
            return
        n_decode = ctx.T if ctx.decode_only else ctx.n_decode
        if n_decode:
            ops.diff_attention_decode(
                q, view.k_cache, view.v_cache, None if ctx.decode_only else ctx.decode_rows,
                n_decode, ctx.seq_of_token, ctx.positions, tables, out, self.H, s.softmax_scale,
                dc, ctx.max_ctx_len if ctx.decode_only else ctx.max_decode_ctx, ctx.err)
        if ctx.n_prefill and not ctx.decode_only:
            ops.diff_attention_prefill(q, view.k_cache, view.v_cache, ctx.prefill_items,
                                       ctx.n_prefill, ctx.max_prefill_rows, tables, out, self.H,
                                       s.softmax_scale, dc, ctx.err, max_ctx=ctx.max_ctx_len)


register_mixer("differential_attention", DifferentialAttention)
