// What the differential attention kernels share (attention_diff.cu says what is computed).
#pragma once
#include "common.cuh"

// How two maps become a head's output: o = a1 - lambda a2, o <- o / sqrt(mean(o^2) + eps) times
// out_factor, times sigmoid(gate) element by element (gate null: not; a row every `gate_stride`
// elements of the activation type, head h's at columns h dv ..).  q at position p counts
// 1 + temp_coef ln(floor((p + 1) / temp_every) + 1) times (temp_coef 0: once).
struct BfDiffArgs {
  const void* gate;
  long long gate_stride;
  float lambda, eps, out_factor, temp_coef;
  int temp_every;
};

__device__ __forceinline__ float bf_query_temperature(int p, float coef, int every) {
  return coef == 0.f ? 1.f : 1.f + coef * logf((float)((p + 1) / every + 1));
}
// for bfloat16 results (see bf_silu_fast's remark on the fast instructions' error)
__device__ __forceinline__ float bf_sigmoid_fast(float z) {
  return __fdividef(1.f, 1.f + __expf(-z));
}

// Partial results of shares of the keys made one: defined in attention_diff.cu.  part_o
// [rows][nh][2][splits][dv] unnormalised, part_ml [rows][nh][2][splits][2] the base-2 exponent
// reference (minus infinity: nothing in this share) and the sum.
//
// _rows: partial row r belongs to token rows[r] (null: r), whose splits are those of 128 keys up
// to its position.  _items: (request, first token row, rows, first position) portions, every row
// with the same number of splits, partial rows by token row.
int bf_diff_attention_merge_rows(const float* part_o, const float* part_ml, const int* rows,
                                 const int* positions, void* out, int n_rows, int nh, int dv,
                                 int max_splits, long long out_stride, const BfDiffArgs& dd,
                                 cudaStream_t stream);
int bf_diff_attention_merge_items(const float* part_o, const float* part_ml, const int* items,
                                  int n_items, int max_rows, void* out, int nh, int dv,
                                  int splits, long long out_stride, const BfDiffArgs& dd,
                                  cudaStream_t stream);
