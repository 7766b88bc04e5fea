// Norm without statistics over the float residual stream, fused with the stream's pending adds:
//   v = x + d1 + d2 + bias;   y = tanh(alpha v) w + b
// (alpha one number; `bias` the bias of the product that made a pending add), and the row pair
// that a pass over a run of layers starts from:
//   pair[t] = [x + d1 + d2 + bias | table[ids[t]] scale].
//
// Nothing couples the columns of a row, so the grid is a flat walk over pieces of eight
// neighbouring columns (one where the sizes or addresses do not allow it).  The stream is
// written back when asked.  `rows` picks the rows to norm (the output is then packed).
#include "common.cuh"

__device__ __forceinline__ void tn_ld8(const float* p, float (&v)[8]) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void tn_ld8(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 q = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&q);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 f = __bfloat1622float2(h[j]);
    v[2 * j] = f.x;
    v[2 * j + 1] = f.y;
  }
}
__device__ __forceinline__ void tn_st8(float* p, const float (&v)[8]) {
  reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void tn_st8(__nv_bfloat16* p, const float (&v)[8]) {
  uint4 q;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&q);
#pragma unroll
  for (int j = 0; j < 4; ++j) h[j] = __floats2bfloat162_rn(v[2 * j], v[2 * j + 1]);
  *reinterpret_cast<uint4*>(p) = q;
}
// N neighbouring values: eight with wide accesses, or one
template <int N, typename A>
__device__ __forceinline__ void tn_ld(const A* p, float (&v)[N]) {
  if constexpr (N == 8) tn_ld8(p, v);
  else v[0] = bf_ld(p);
}
template <int N, typename A>
__device__ __forceinline__ void tn_st(A* p, const float (&v)[N]) {
  if constexpr (N == 8) tn_st8(p, v);
  else bf_st(p, v[0]);
}

// v += what is pending at `at` (a place of the stream) and column c
template <int N, typename A>
__device__ __forceinline__ void tn_fold(float (&v)[N], const A* d1, const A* d2,
                                        const float* bias, size_t at, int c) {
  float e[N];
  if (d1) {
    tn_ld<N>(d1 + at, e);
#pragma unroll
    for (int j = 0; j < N; ++j) v[j] += e[j];
  }
  if (d2) {
    tn_ld<N>(d2 + at, e);
#pragma unroll
    for (int j = 0; j < N; ++j) v[j] += e[j];
  }
  if (bias) {
    tn_ld<N>(bias + c, e);
#pragma unroll
    for (int j = 0; j < N; ++j) v[j] += e[j];
  }
}

template <int N, typename A>
__global__ void __launch_bounds__(256) add_tanh_norm_kernel(
    float* __restrict__ resid, const A* __restrict__ d1, const A* __restrict__ d2,
    const float* __restrict__ bias, float alpha, const float* __restrict__ w,
    const float* __restrict__ b, A* __restrict__ out, const int* __restrict__ rows, int n_rows,
    int H, int write_back) {
  bf_pdl_trigger();
  bf_pdl_wait();
  const int per = H / N;
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= (long long)n_rows * per) return;
  const int i = (int)(idx / per), c = (int)(idx - (long long)i * per) * N;
  const int r = rows ? rows[i] : i;
  const size_t at = (size_t)r * H + c;
  float v[N], wv[N], bv[N];
  tn_ld<N>(resid + at, v);
  tn_ld<N>(w + c, wv);
  if (b) tn_ld<N>(b + c, bv);
  tn_fold<N>(v, d1, d2, bias, at, c);
  if (write_back && (d1 || d2 || bias)) tn_st<N>(resid + at, v);
#pragma unroll
  for (int j = 0; j < N; ++j) v[j] = tanhf(alpha * v[j]) * wv[j] + (b ? bv[j] : 0.f);
  tn_st<N>(out + (size_t)i * H + c, v);
}

template <int N, typename A>
__global__ void __launch_bounds__(256) stream_pair_kernel(
    const float* __restrict__ resid, const A* __restrict__ d1, const A* __restrict__ d2,
    const float* __restrict__ bias, const A* __restrict__ table, const int* __restrict__ ids,
    int vocab, float scale, A* __restrict__ pair, int T, int H, int* __restrict__ err) {
  bf_pdl_trigger();
  bf_pdl_wait();
  const int per = H / N;
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= (long long)T * per) return;
  const int t = (int)(idx / per), c = (int)(idx - (long long)t * per) * N;
  const size_t at = (size_t)t * H + c;
  float v[N], e[N];
  tn_ld<N>(resid + at, v);
  tn_fold<N>(v, d1, d2, bias, at, c);
  A* o = pair + (size_t)t * 2 * H + c;
  tn_st<N>(o, v);
#pragma unroll
  for (int j = 0; j < N; ++j) e[j] = 0.f;
  const int id = ids[t];
  if (id < 0 || id >= vocab) {
    if (c == 0) atomicOr(err, BF_ERR_TOKEN_ID);
  } else {
    tn_ld<N>(table + (size_t)id * H + c, e);
  }
#pragma unroll
  for (int j = 0; j < N; ++j) e[j] *= scale;
  tn_st<N>(o + H, e);
}

static inline bool tn_aligned(const void* a, const void* b, const void* c, const void* d,
                              const void* e, const void* f, const void* g) {
  return ((((uintptr_t)a) | ((uintptr_t)b) | ((uintptr_t)c) | ((uintptr_t)d) | ((uintptr_t)e) |
           ((uintptr_t)f) | ((uintptr_t)g)) & 15) == 0;
}

BF_EXPORT int bf_add_tanh_norm(float* resid, const void* d1, const void* d2, const float* bias,
                               float alpha, const float* w, const float* b, void* out,
                               const int* rows, int n_rows, int H, int act_dtype, int write_back,
                               cudaStream_t stream) {
  if (n_rows <= 0 || H <= 0) return 0;
  const bool vec = H % 8 == 0 && tn_aligned(resid, d1, d2, bias, w, b, out);
  const int threads = 256;
  const long long n = (long long)n_rows * (vec ? H / 8 : H);
  const unsigned blocks = (unsigned)((n + threads - 1) / threads);
#define TN_GO(N, A)                                                                            \
  return bf_launch_pdl(add_tanh_norm_kernel<N, A>, dim3(blocks), dim3(threads), 0, stream,     \
                       resid, (const A*)d1, (const A*)d2, bias, alpha, w, b, (A*)out, rows,    \
                       n_rows, H, write_back)
  if (act_dtype == BF_DTYPE_F32) {
    if (vec) TN_GO(8, float);
    TN_GO(1, float);
  }
  if (vec) TN_GO(8, __nv_bfloat16);
  TN_GO(1, __nv_bfloat16);
#undef TN_GO
}

// The table's type is the activations' (a float engine holds it in float).
BF_EXPORT int bf_stream_pair(const float* resid, const void* d1, const void* d2,
                             const float* bias, const void* table, const int* ids, int vocab,
                             float scale, void* pair, int T, int H, int act_dtype, int* err,
                             cudaStream_t stream) {
  if (T <= 0 || H <= 0) return 0;
  const bool vec = H % 8 == 0 && tn_aligned(resid, d1, d2, bias, table, pair, nullptr);
  const int threads = 256;
  const long long n = (long long)T * (vec ? H / 8 : H);
  const unsigned blocks = (unsigned)((n + threads - 1) / threads);
#define SP_GO(N, A)                                                                            \
  return bf_launch_pdl(stream_pair_kernel<N, A>, dim3(blocks), dim3(threads), 0, stream,    \
                       resid, (const A*)d1, (const A*)d2, bias, (const A*)table, ids, vocab,   \
                       scale, (A*)pair, T, H, err)
  if (act_dtype == BF_DTYPE_F32) {
    if (vec) SP_GO(8, float);
    SP_GO(1, float);
  }
  if (vec) SP_GO(8, __nv_bfloat16);
  SP_GO(1, __nv_bfloat16);
#undef SP_GO
}
