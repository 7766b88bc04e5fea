// Activations of gated feed-forwards, act(gate) * up, shared by the activation kernels and the
// products that apply one in their epilogue.
//
// ACT 0: silu, g / (1 + exp(-g)), times up.
// ACT 1: the tanh form of gelu in silu's place,
//   gelu(g) = 0.5 g (1 + tanh(sqrt(2/pi) (g + 0.044715 g^3))).
// ACT 2: clamped, with three constants: g = min(gate, limit), u = clamp(up, -limit, limit),
//   g sigmoid(slope g) (u + up_offset).
#pragma once
#include "common.cuh"

#define BF_ACT_SILU 0
#define BF_ACT_GELU_TANH 1
#define BF_ACT_CLAMPED 2
struct BfGateConst {
  float limit, slope, up_offset;
};
// Outputs that belong to the experts of a mixture, `ff` neighbouring ones each and the shared
// expert's behind them: output o of token t counts w[t, expert(o)] times (w [T, cols]; the shared
// expert counts w[t, experts] times with `shared_gate`, else once), and the shared expert's clamped
// activation has a limit of its own.  w null: no mixture.
struct BfMixture {
  const float* w;
  int cols, experts, ff, shared_gate;
  float shared_limit;
};
// the weight of output o for token t; k becomes the constants of o's activation
__device__ __forceinline__ float bf_mix_weight(const BfMixture& m, int t, int o, BfGateConst& k) {
  if (o < m.experts * m.ff) return m.w[(size_t)t * m.cols + o / m.ff];
  k.limit = m.shared_limit;
  return m.shared_gate ? m.w[(size_t)t * m.cols + m.experts] : 1.f;
}
template <int ACT>
__device__ __forceinline__ float bf_gate_mul(float g, float u, const BfGateConst& k) {
  if (ACT == BF_ACT_CLAMPED) {
    g = fminf(g, k.limit);
    u = fminf(fmaxf(u, -k.limit), k.limit) + k.up_offset;
    return g / (1.f + expf(-k.slope * g)) * u;
  }
  if (ACT == BF_ACT_GELU_TANH)
    return 0.5f * g * (1.f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g))) * u;
  return g / (1.f + expf(-g)) * u;
}

// silu for the bf16 kernels: float arithmetic with the hardware's exp2 and reciprocal
// approximations (relative error about 2^-21, far inside the bf16 result's 2^-9).  With the
// accurate expf and division the bf16 kernel was bound by arithmetic, not by memory.
__device__ __forceinline__ float bf_silu_fast(float g) { return __fdividef(g, 1.f + __expf(-g)); }
// ... and gelu's tanh form the same way: 0.5 g (1 + tanh(z)) = g / (1 + exp(-2 z))
template <int ACT>
__device__ __forceinline__ float bf_gate_mul_fast(float g, float u, const BfGateConst& k) {
  if (ACT == BF_ACT_CLAMPED) {
    g = fminf(g, k.limit);
    u = fminf(fmaxf(u, -k.limit), k.limit) + k.up_offset;
    return __fdividef(g, 1.f + __expf(-k.slope * g)) * u;
  }
  if (ACT == BF_ACT_GELU_TANH) {
    const float z = 0.7978845608028654f * (g + 0.044715f * g * g * g);
    return __fdividef(g, 1.f + __expf(-2.f * z)) * u;
  }
  return bf_silu_fast(g) * u;
}
