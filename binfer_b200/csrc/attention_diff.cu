// Differential attention over the paged cache: a head is the normed difference of two causal
// softmax maps over the same values.
//
// A query head and a key head hold two vectors of d numbers side by side, one per map; with a1
// and a2 the outputs of the two maps (values of dv numbers) a head's result is
//   o = a1 - lambda a2;   o <- o / sqrt(mean(o^2) + eps) * out_factor * sigmoid(gate)
// (the mean over the dv values; the gate element by element, optional).  A cached key row is
// the 2 d numbers of both maps.  q at position p counts 1 + temp_coef ln(floor((p + 1) /
// temp_every) + 1) times: the factor rides on the score scale, in float.
//
// Here: the store of a step's keys and values into the pages; the kernel for any sizes, which
// is the whole 32-bit path and the fallback in bfloat16; and the merge of shares of the keys.
// The tensor-core kernels are in attention_diff_mma.cu (mma.sync, prompt portions and single
// tokens), attention_prefill_umma2.cu (tcgen05, d 64 and dv 128) and
// attention_decode_persistent.cu (single tokens, 2 d = dv); they share the merge.
#include <float.h>

#include "attention_diff.cuh"
#include "common.cuh"

// ---------------------------------------------------------------- keys and values to pages
// Token t's row of `proj` (stride elements) holds nkv key heads of dk at k_off and nkv value
// heads of dv at v_off; they go to page slot / page_size, place slot % page_size.  A thread
// moves one piece of VEC elements (pieces do not cross heads).
template <typename A, int VEC>
__global__ void kv_store_kernel(const A* __restrict__ proj, long long stride, int k_off, int v_off,
                                const int* __restrict__ slots, A* __restrict__ k_cache,
                                A* __restrict__ v_cache, int T, int nkv, int dk, int dv,
                                int page_size, long long num_slots, int* __restrict__ err) {
  bf_pdl_trigger();
  bf_pdl_wait();
  const int kp = nkv * dk / VEC, per = kp + nkv * dv / VEC;
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)T * per) return;
  const int t = (int)(i / per);
  int c = (int)(i - (long long)t * per);
  const long long s = slots[t];
  if (s < 0 || s >= num_slots) {
    if (c == 0) atomicOr(err, BF_ERR_SLOT);
    return;
  }
  const bool is_v = c >= kp;
  if (is_v) c -= kp;
  c *= VEC;
  const int d = is_v ? dv : dk;
  const int g = c / d, col = c - g * d;
  const long long page = s / page_size, off = s - page * page_size;
  const A* src = proj + (size_t)t * stride + (is_v ? v_off : k_off) + c;
  A* dst = (is_v ? v_cache : k_cache) + ((page * nkv + g) * page_size + off) * d + col;
  if (VEC * sizeof(A) == 16)
    *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(src);
  else
    *dst = *src;
}

BF_EXPORT int bf_kv_store(const void* proj, long long stride, int k_off, int v_off,
                          const int* slots, void* k_cache, void* v_cache, int T, int nkv, int dk,
                          int dv, int page_size, long long num_slots, int act_dtype, int* err,
                          cudaStream_t stream) {
  if (T <= 0) return 0;
  if (nkv <= 0 || dk <= 0 || dv <= 0) return (int)cudaErrorInvalidValue;
  const bool f32 = act_dtype == BF_DTYPE_F32;
  const int vec = f32 ? 4 : 8;
  const bool ok16 = dk % vec == 0 && dv % vec == 0 && stride % vec == 0 && k_off % vec == 0 &&
                    v_off % vec == 0 &&
                    (((uintptr_t)proj | (uintptr_t)k_cache | (uintptr_t)v_cache) & 15) == 0;
  const long long n = (long long)T * nkv * (dk + dv) / (ok16 ? vec : 1);
  const unsigned blocks = (unsigned)((n + 255) / 256);
#define KVS_GO(AT, V)                                                                        \
  return bf_launch_pdl(kv_store_kernel<AT, V>, dim3(blocks), dim3(256), 0, stream,           \
                       (const AT*)proj, stride, k_off, v_off, slots, (AT*)k_cache,           \
                       (AT*)v_cache, T, nkv, dk, dv, page_size, num_slots, err)
  if (f32) {
    if (ok16) KVS_GO(float, 4);
    KVS_GO(float, 1);
  }
  if (ok16) KVS_GO(__nv_bfloat16, 8);
  KVS_GO(__nv_bfloat16, 1);
#undef KVS_GO
}

// ------------------------------------------------------------------------- any sizes
// One warp per (token, head).  Keys are walked in tiles of 32 counted from position 0, a key a
// lane, both maps' scores from one walk over the key row; two online softmaxes in float; each
// value row is fetched once for both maps.  The order of every sum depends on the position
// alone, never on how the tokens were cut into steps or on what else is in the batch.
template <typename A, int ACC>             // value size <= 32 * ACC
__global__ void diff_attention_generic_kernel(
    const A* __restrict__ q, long long q_stride, const A* __restrict__ k_cache,
    const A* __restrict__ v_cache, const int* __restrict__ seq_of_token,
    const int* __restrict__ positions, const int* __restrict__ block_tables, int table_stride,
    A* __restrict__ out, long long out_stride, int nh, int nkv, int d, int dv, int page_size,
    int num_pages, float scale, int* __restrict__ err, BfDiffArgs dd) {
  extern __shared__ float sh[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int warps = blockDim.x >> 5;
  const int t = blockIdx.x;
  const int h = blockIdx.y * warps + warp;
  if (h >= nh) return;
  const int g = h / (nh / nkv);
  float* qs = sh + (size_t)warp * 2 * d;
  const int p = positions[t];
  const A* qrow = q + (size_t)t * q_stride + (size_t)h * 2 * d;
  const float f = scale * bf_query_temperature(p, dd.temp_coef, dd.temp_every);
  for (int i = lane; i < 2 * d; i += 32) qs[i] = bf_ld(qrow + i) * f;
  __syncwarp();
  const int* table = block_tables + (size_t)seq_of_token[t] * table_stride;

  float m[2] = {-FLT_MAX, -FLT_MAX}, l[2] = {0.f, 0.f};
  float acc[2][ACC];
#pragma unroll
  for (int c = 0; c < ACC; ++c) acc[0][c] = acc[1][c] = 0.f;
  for (int tile = 0; tile <= (p >> 5); ++tile) {
    const int j = (tile << 5) + lane;
    bool valid = j <= p;
    long long row = 0;
    if (valid) {
      const int lp = j / page_size;
      const int page = table[lp];
      if (page < 0 || page >= num_pages) {
        atomicOr(err, BF_ERR_PAGE);
        valid = false;
      } else {
        row = ((long long)page * nkv + g) * page_size + (j - lp * page_size);
      }
    }
    float pj[2] = {0.f, 0.f};
    float s[2] = {-FLT_MAX, -FLT_MAX};
    if (valid) {
      const A* kr = k_cache + row * 2 * d;
#pragma unroll
      for (int mp = 0; mp < 2; ++mp) {
        float a = 0.f;
#pragma unroll 8
        for (int i = 0; i < d; ++i) a += qs[mp * d + i] * bf_ld(kr + mp * d + i);
        s[mp] = a;
      }
    }
#pragma unroll
    for (int mp = 0; mp < 2; ++mp) {
      const float m_new = fmaxf(m[mp], warp_max(s[mp]));
      const float corr = expf(m[mp] - m_new);
      pj[mp] = valid ? expf(s[mp] - m_new) : 0.f;
      l[mp] = l[mp] * corr + warp_sum(pj[mp]);
      m[mp] = m_new;
#pragma unroll
      for (int c = 0; c < ACC; ++c) acc[mp][c] *= corr;
    }
    const unsigned live = __ballot_sync(0xffffffffu, valid);
    for (int jj = 0; jj < 32; ++jj) {
      if (!((live >> jj) & 1u)) continue;
      const float p0 = __shfl_sync(0xffffffffu, pj[0], jj);
      const float p1 = __shfl_sync(0xffffffffu, pj[1], jj);
      const long long rb = __shfl_sync(0xffffffffu, row, jj);
      const A* vr = v_cache + rb * dv;
#pragma unroll
      for (int c = 0; c < ACC; ++c) {
        const int i = lane + 32 * c;
        if (i < dv) {
          const float v = bf_ld(vr + i);
          acc[0][c] += p0 * v;
          acc[1][c] += p1 * v;
        }
      }
    }
  }
  const float inv0 = 1.f / l[0], inv1 = dd.lambda / l[1];
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < ACC; ++c) {
    const float o = lane + 32 * c < dv ? acc[0][c] * inv0 - acc[1][c] * inv1 : 0.f;
    acc[0][c] = o;
    ss += o * o;
  }
  const float r = rsqrtf(warp_sum(ss) / (float)dv + dd.eps) * dd.out_factor;
  A* o = out + (size_t)t * out_stride + (size_t)h * dv;
  const A* gate = dd.gate ? (const A*)dd.gate + (size_t)t * dd.gate_stride + (size_t)h * dv
                          : nullptr;
#pragma unroll
  for (int c = 0; c < ACC; ++c) {
    const int i = lane + 32 * c;
    if (i < dv) {
      float v = acc[0][c] * r;
      if (gate) v /= 1.f + expf(-bf_ld(gate + i));
      bf_st(o + i, v);
    }
  }
}

BF_EXPORT int bf_diff_attention_generic(
    const void* q, long long q_stride, const void* k_cache, const void* v_cache,
    const int* seq_of_token, const int* positions, const int* block_tables, int table_stride,
    void* out, long long out_stride, int T, int nh, int nkv, int d, int dv, int page_size,
    int num_pages, float scale, int act_dtype, int* err, const void* gate, long long gate_stride,
    float lambda, float eps, float out_factor, float temp_coef, int temp_every,
    cudaStream_t stream) {
  if (T <= 0) return 0;
  if (d <= 0 || d > 512 || dv <= 0 || dv > 512 || nkv <= 0 || nh % nkv || temp_every < 1)
    return (int)cudaErrorInvalidValue;
  const BfDiffArgs dd = {gate, gate_stride, lambda, eps, out_factor, temp_coef, temp_every};
  const int warps = 4;
  dim3 grid(T, (nh + warps - 1) / warps);
  const size_t smem = (size_t)warps * 2 * d * sizeof(float);
#define DG_GO(AT, ACC)                                                                         \
  diff_attention_generic_kernel<AT, ACC><<<grid, warps * 32, smem, stream>>>(                  \
      (const AT*)q, q_stride, (const AT*)k_cache, (const AT*)v_cache, seq_of_token, positions, \
      block_tables, table_stride, (AT*)out, out_stride, nh, nkv, d, dv, page_size, num_pages,  \
      scale, err, dd)
  if (act_dtype == BF_DTYPE_F32) {
    if (dv <= 128) DG_GO(float, 4); else DG_GO(float, 16);
  } else {
    if (dv <= 128) DG_GO(__nv_bfloat16, 4); else DG_GO(__nv_bfloat16, 16);
  }
#undef DG_GO
  return bf_launch_status();
}

// --------------------------------------------------------------- shares of the keys made one
// A block of eight warps per (row, head), four per map: a warp sums every fourth share of its
// map, a lane four neighbouring columns, eight shares' loads in flight before anything else is
// known; the four sums are then added in order and the two maps become the head's output.
#define DM_WARPS 4
#define DM_AHEAD 8

__global__ void __launch_bounds__(2 * DM_WARPS * 32) diff_merge_kernel(
    const float* __restrict__ part_o, const float* __restrict__ part_ml,
    const int* __restrict__ rows, const int* __restrict__ positions,
    const int* __restrict__ items, __nv_bfloat16* __restrict__ out, int nh, int dv,
    int max_splits, int fixed, long long out_stride, BfDiffArgs dd) {
  extern __shared__ __align__(16) float sh[];   // [2][4][dv] the warps' sums, [2][max_splits] weights
  __shared__ float scratch[33];
  bf_pdl_trigger();
  bf_pdl_wait();
  const int h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int mp = warp / DM_WARPS, wm = warp % DM_WARPS;
  int r, t, n;
  if (items) {                             // a portion's row; its partials lie by token row
    const int* it = items + 4 * blockIdx.z;
    if ((int)blockIdx.x >= it[2]) return;
    r = t = it[1] + blockIdx.x;
    n = fixed;
  } else {
    r = blockIdx.x;
    t = rows ? rows[r] : r;
    n = min(max_splits, positions[t] / 128 + 1);
  }
  float* sums = sh + (size_t)mp * DM_WARPS * dv;
  float* wgt = sh + (size_t)2 * DM_WARPS * dv + (size_t)mp * max_splits;
  const size_t at = (((size_t)r * nh + h) * 2 + mp) * max_splits;
  const float4* po = reinterpret_cast<const float4*>(part_o + at * dv);
  const int dv4 = dv >> 2;
  float4 x[DM_AHEAD];                      // the first shares of the lane's first columns
#pragma unroll
  for (int u = 0; u < DM_AHEAD; ++u) {
    const int s = wm + DM_WARPS * u;
    x[u] = s < n && lane < dv4 ? po[(size_t)s * dv4 + lane] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  // every warp works out the maximum and the sum of its map; the map's first writes the weights
  const float2* ml = reinterpret_cast<const float2*>(part_ml) + at;
  const float2 mine = lane < n ? ml[lane] : make_float2(-INFINITY, 0.f);
  float M = mine.x;
  for (int s = lane + 32; s < n; s += 32) M = fmaxf(M, ml[s].x);
  M = warp_max(M);
  float L = mine.x == -INFINITY ? 0.f : mine.y * exp2f(mine.x - M);
  for (int s = lane + 32; s < n; s += 32)
    if (ml[s].x != -INFINITY) L += ml[s].y * exp2f(ml[s].x - M);
  L = warp_sum(L);
  if (wm == 0) {
    const float inv = L > 0.f ? 1.f / L : 0.f;
    for (int s = lane; s < n; s += 32) {
      const float ms = s < 32 ? mine.x : ml[s].x;
      wgt[s] = ms == -INFINITY ? 0.f : exp2f(ms - M) * inv;
    }
  }
  __syncthreads();
  for (int c = lane; c < dv4; c += 32) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s0 = wm; s0 < n; s0 += DM_WARPS * DM_AHEAD) {
      if (s0 != wm || c != lane) {
#pragma unroll
        for (int u = 0; u < DM_AHEAD; ++u) {
          const int s = s0 + DM_WARPS * u;
          if (s < n) x[u] = po[(size_t)s * dv4 + c];
        }
      }
#pragma unroll
      for (int u = 0; u < DM_AHEAD; ++u) {
        const int s = s0 + DM_WARPS * u;
        const float w = s < n ? wgt[s] : 0.f;
        if (w != 0.f) {                    // (a share without keys has left nothing)
          v.x += x[u].x * w;
          v.y += x[u].y * w;
          v.z += x[u].z * w;
          v.w += x[u].w * w;
        }
      }
    }
    reinterpret_cast<float4*>(sums + (size_t)wm * dv)[c] = v;
  }
  __syncthreads();
  float* a1 = sh;
  const float* a2 = sh + (size_t)DM_WARPS * dv;
  float ss = 0.f;
  for (int c = threadIdx.x; c < dv; c += blockDim.x) {
    float o1 = 0.f, o2 = 0.f;
#pragma unroll
    for (int w = 0; w < DM_WARPS; ++w) {
      o1 += a1[w * dv + c];
      o2 += a2[w * dv + c];
    }
    const float o = o1 - dd.lambda * o2;
    a1[c] = o;                             // (this thread's own column)
    ss += o * o;
  }
  ss = block_sum(ss, scratch);
  const float f = rsqrtf(ss / (float)dv + dd.eps) * dd.out_factor;
  __nv_bfloat16* o = out + (size_t)t * out_stride + (size_t)h * dv;
  const __nv_bfloat16* gate =
      dd.gate ? (const __nv_bfloat16*)dd.gate + (size_t)t * dd.gate_stride + (size_t)h * dv
              : nullptr;
  for (int c = threadIdx.x; c < dv; c += blockDim.x) {
    float v = a1[c] * f;
    if (gate) v *= bf_sigmoid_fast(__bfloat162float(gate[c]));
    o[c] = __float2bfloat16_rn(v);
  }
}

static int diff_merge(dim3 grid, const float* part_o, const float* part_ml, const int* rows,
                      const int* positions, const int* items, void* out, int nh, int dv,
                      int max_splits, int fixed, long long out_stride, const BfDiffArgs& dd,
                      cudaStream_t stream) {
  const size_t smem = (size_t)2 * (max_splits + DM_WARPS * dv) * sizeof(float);
  if (smem > 200 * 1024 || dv <= 0 || dv % 4 || max_splits <= 0 || ((uintptr_t)part_o & 15) ||
      ((uintptr_t)part_ml & 7)) return (int)cudaErrorInvalidValue;
  if (smem > 48 * 1024) {
    static size_t configured[BF_MAX_DEVICES];
    size_t& c = configured[bf_current_device()];
    if (c < smem) {
      const cudaError_t e = cudaFuncSetAttribute(
          diff_merge_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
      if (e != cudaSuccess) return (int)e;
      c = 200 * 1024;
    }
  }
  return bf_launch_pdl(diff_merge_kernel, grid, dim3(2 * DM_WARPS * 32), smem, stream, part_o, part_ml,
                       rows, positions, items, (__nv_bfloat16*)out, nh, dv, max_splits, fixed,
                       out_stride, dd);
}

int bf_diff_attention_merge_rows(const float* part_o, const float* part_ml, const int* rows,
                                 const int* positions, void* out, int n_rows, int nh, int dv,
                                 int max_splits, long long out_stride, const BfDiffArgs& dd,
                                 cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  return diff_merge(dim3(n_rows, nh), part_o, part_ml, rows, positions, nullptr, out, nh, dv,
                    max_splits, 0, out_stride, dd, stream);
}

int bf_diff_attention_merge_items(const float* part_o, const float* part_ml, const int* items,
                                  int n_items, int max_rows, void* out, int nh, int dv,
                                  int splits, long long out_stride, const BfDiffArgs& dd,
                                  cudaStream_t stream) {
  if (n_items <= 0 || max_rows <= 0) return 0;
  return diff_merge(dim3(max_rows, nh, n_items), part_o, part_ml, nullptr, nullptr, items, out,
                    nh, dv, splits, splits, out_stride, dd, stream);
}
