// Differential attention (attention_diff.cu says what it computes) on the tensor cores for
// bfloat16 heads of d key columns a map and dv values, both multiples of 16 up to 128.
//
// Prompt portions: a CTA of four warps takes 64 rows of one portion and one key/value head, a
// row being a (token, query head of the group) pair, tokens in order and the group's heads side
// by side.  It walks the keys in tiles of 64: K rows (both maps side by side) and V rows come
// through the block table by asynchronous copies into one of two stages; per tile and map S = Q
// K^T by mma.sync m16n8k16, each row masks by its own position, online softmax in float in
// base 2, P in bfloat16 straight from the accumulators; each V fragment is then read once for
// both maps' O += P V.  A row's values lie in the four lanes of a quad, so the epilogue
// (difference, root mean square, gate) needs two shuffles.
//
// Single tokens: a warp takes one share of 128 keys for up to 16 heads of a group and leaves a
// partial result per map for the merge kernel; the four warps of a CTA take neighbouring shares
// and never wait for each other.  A warp's tiles of 16 keys come by bulk copies, a row a lane (16
// key rows, 16 value rows), three tiles under way; two CTAs fit an SM.
//
// q is read from the rows of the stacked projection; the query temperature rides on the scale.
#include <float.h>

#include "attention_diff.cuh"
#include "common.cuh"
#include "mma_utils.cuh"
#include "tma_utils.cuh"

#define DA_ROWS 64
#define DA_KEYS 64
#define DA_THREADS 128
#define DA_SHARE 128        // keys a warp takes while decoding
#define DA_DKEYS 16         // ... in tiles of this many
#define DA_DSTAGES 3        // ... of which this many are under way

__device__ __forceinline__ float da_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// A walk over the 16-byte pieces of a tile's rows by `n` threads: the piece of this thread at
// first and the step to its next one, so that the loop divides nothing.
struct DaWalk {
  int row, c, chunks, drow, dc;
};
__device__ __forceinline__ DaWalk da_walk(int d, int id, int n) {
  DaWalk w;
  w.chunks = d >> 3;
  w.row = id / w.chunks;
  w.c = id - w.row * w.chunks;
  w.drow = n / w.chunks;
  w.dc = n - w.drow * w.chunks;
  return w;
}
// `rows` cache rows on their way into a shared tile: tile row r is the cache's row at(r) (-1:
// none, the tile's row is zeroed: a copy of 0 bytes reads nothing).  Every thread of a warp
// makes as many steps as any other (`at` may be a shuffle).
template <typename AtFn>
__device__ __forceinline__ void da_load_rows(__nv_bfloat16* tile, int pitch,
                                             const __nv_bfloat16* __restrict__ cache, int rows,
                                             DaWalk w, int steps, AtFn at) {
#pragma unroll 4
  for (int k = 0; k < steps; ++k) {
    const int e = at(min(w.row, rows - 1));
    if (w.row < rows)
      cp_async16(tile + w.row * pitch + w.c * 8,
                 cache + (e >= 0 ? ((size_t)e * w.chunks + w.c) * 8 : 0), e >= 0 ? 16 : 0);
    w.row += w.drow;
    w.c += w.dc;
    if (w.c >= w.chunks) {
      w.c -= w.chunks;
      ++w.row;
    }
  }
}
// The cache row of key e of a request for kv head g, or -1 beyond `limit` (or a bad page).
__device__ __forceinline__ int da_cache_row(const int* __restrict__ table, int e, int limit,
                                            int nkv, int g, int page_size, int num_pages,
                                            int* __restrict__ err) {
  if (e >= limit) return -1;
  const int lp = e / page_size;
  const int page = table[lp];
  if (page < 0 || page >= num_pages) {
    atomicOr(err, BF_ERR_PAGE);
    return -1;
  }
  return (page * nkv + g) * page_size + (e - lp * page_size);
}

// One map of one key tile: S = Q K^T for the warp's 16 rows and KT keys, the mask, the online
// softmax; the probabilities leave as A fragments.  Q at `qt` (the warp's first row, this map's
// first column), K at `kt` (this map's first column).  `rel` per row: its last visible key minus
// the tile's first; whole: every row sees every key.
template <int KT>
__device__ __forceinline__ void da_scores(const __nv_bfloat16* qt, int pitch_q,
                                          const __nv_bfloat16* kt, int pitch_k, int d, int lane,
                                          const int (&rel)[2], bool whole, const float (&sc)[2],
                                          float (&m)[2], float (&l)[2], float (&corr)[2],
                                          uint32_t (&pa)[KT / 16][4]) {
  float s[KT / 8][4];
#pragma unroll
  for (int n = 0; n < KT / 8; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
#pragma unroll 2
  for (int ks = 0; ks < d; ks += 16) {
    uint32_t qf[4];
    ldmatrix_x4(qf, qt + (size_t)(lane & 15) * pitch_q + ks + (lane >> 4) * 8);
#pragma unroll
    for (int np = 0; np < KT / 16; ++np) {
      uint32_t kb[4];
      ldmatrix_x4(kb, kt + (size_t)(np * 16 + (lane & 7) + ((lane >> 4) << 3)) * pitch_k + ks +
                          ((lane >> 3) & 1) * 8);
      mma_bf16_16816(s[2 * np], qf, kb[0], kb[1]);
      mma_bf16_16816(s[2 * np + 1], qf, kb[2], kb[3]);
    }
  }
  float mx[2] = {-INFINITY, -INFINITY};
  if (!whole) {
#pragma unroll
    for (int n = 0; n < KT / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (n * 8 + 2 * (lane & 3) + (e & 1) > rel[e >> 1]) s[n][e] = -INFINITY;
  }
#pragma unroll
  for (int n = 0; n < KT / 8; ++n) {
    mx[0] = fmaxf(mx[0], fmaxf(s[n][0], s[n][1]));
    mx[1] = fmaxf(mx[1], fmaxf(s[n][2], s[n][3]));
  }
  float ref[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
    mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
    // the reference follows the maximum only when that has grown by more than 8 (a factor of
    // 256 in the probabilities, harmless in bfloat16 and float), so O is rarely rescaled
    const float top = mx[i] * sc[i];                     // the factor is positive
    const float m_new = top > m[i] + 8.f ? top : m[i];
    ref[i] = m_new == -INFINITY ? 0.f : m_new;           // a row that has seen nothing yet
    corr[i] = da_ex2(m[i] - ref[i]);
    m[i] = m_new;
    l[i] *= corr[i];
  }
#pragma unroll
  for (int kk = 0; kk < KT / 16; ++kk) {
    float p[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const int n = 2 * kk + (e >> 2), i = (e >> 1) & 1;
      p[e] = da_ex2(fmaf(s[n][e & 3], sc[i], -ref[i]));
      l[i] += p[e];
    }
    pa[kk][0] = pack_bf16(p[0], p[1]);
    pa[kk][1] = pack_bf16(p[2], p[3]);
    pa[kk][2] = pack_bf16(p[4], p[5]);
    pa[kk][3] = pack_bf16(p[6], p[7]);
  }
}

// O_m <- corr_m O_m + P_m V for both maps, a V fragment read once for the two.
template <int KT, int DVT>
__device__ __forceinline__ void da_values(const __nv_bfloat16* vt, int pitch_v, int dv, int lane,
                                          const uint32_t (&pa)[2][KT / 16][4],
                                          const float (&corr)[2][2], float (&o)[2][DVT][4]) {
  // (most tiles move no row's reference: the factors are one)
  if (__any_sync(0xffffffffu, corr[0][0] != 1.f || corr[0][1] != 1.f || corr[1][0] != 1.f ||
                                  corr[1][1] != 1.f)) {
#pragma unroll
    for (int mp = 0; mp < 2; ++mp)
#pragma unroll
      for (int n = 0; n < DVT; ++n) {
        o[mp][n][0] *= corr[mp][0]; o[mp][n][1] *= corr[mp][0];
        o[mp][n][2] *= corr[mp][1]; o[mp][n][3] *= corr[mp][1];
      }
  }
#pragma unroll
  for (int kk = 0; kk < KT / 16; ++kk) {
#pragma unroll
    for (int np = 0; np < DVT / 2; ++np) {
      if (np * 16 < dv) {
        uint32_t vb[4];
        ldmatrix_x4_trans(vb, vt + (size_t)(kk * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) *
                                       pitch_v + np * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int mp = 0; mp < 2; ++mp) {
          mma_bf16_16816(o[mp][2 * np], pa[mp][kk], vb[0], vb[1]);
          mma_bf16_16816(o[mp][2 * np + 1], pa[mp][kk], vb[2], vb[3]);
        }
      }
    }
  }
}

template <int DVT>                       // value size <= 8 DVT
__global__ void __launch_bounds__(DA_THREADS) diff_prefill_mma_kernel(
    const __nv_bfloat16* __restrict__ q, long long q_stride,
    const __nv_bfloat16* __restrict__ k_cache, const __nv_bfloat16* __restrict__ v_cache,
    const int* __restrict__ items, const int* __restrict__ tables, int table_stride,
    __nv_bfloat16* __restrict__ out, long long out_stride, int nh, int nkv, int d, int dv,
    int page_size, int num_pages, float scale_log2, int* __restrict__ err, BfDiffArgs dd) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __shared__ int where[2][DA_KEYS];
  const int* it = items + 4 * blockIdx.z;
  const int seq = it[0], t0 = it[1], qlen = it[2], pos0 = it[3];
  const int g = blockIdx.y, Gh = nh / nkv;
  const int rows_total = qlen * Gh;
  const int row0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * DA_ROWS;   // the longest blocks first
  if (row0 >= rows_total) return;
  const int pitch_k = 2 * d + 8, pitch_v = dv + 8;
  __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(smem_raw);       // [64][pitch_k]
  __nv_bfloat16* Ks = Qs + (size_t)DA_ROWS * pitch_k;                   // [2][64][pitch_k]
  __nv_bfloat16* Vs = Ks + (size_t)2 * DA_KEYS * pitch_k;               // [2][64][pitch_v]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, wrow = warp * 16;
  const int* table = tables + (size_t)seq * table_stride;

  const int chunks = 2 * d >> 3;
  for (int i = tid; i < DA_ROWS * chunks; i += DA_THREADS) {
    const int r = i / chunks, c = (i - r * chunks) << 3;
    const int row = row0 + r;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (row < rows_total)
      v = *reinterpret_cast<const uint4*>(q + (size_t)(t0 + row / Gh) * q_stride +
                                          (size_t)(g * Gh + row % Gh) * 2 * d + c);
    *reinterpret_cast<uint4*>(Qs + (size_t)r * pitch_k + c) = v;
  }
  int my_p[2];
  float sc[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int row = row0 + wrow + (lane >> 2) + 8 * i;
    my_p[i] = row < rows_total ? pos0 + row / Gh : -1;
    sc[i] = scale_log2 * bf_query_temperature(max(my_p[i], 0), dd.temp_coef, dd.temp_every);
  }
  const int last_row = min(rows_total, row0 + DA_ROWS) - 1;
  const int p_hi = pos0 + last_row / Gh;
  // what the whole warp sees: its first row's position (-1 where a row is missing)
  const int wp_lo = row0 + wrow + 15 < rows_total ? pos0 + (row0 + wrow) / Gh : -1;
  const int n_tiles = p_hi / DA_KEYS + 1;

  float m[2][2], l[2][2], corr[2][2];
  float o[2][DVT][4];
#pragma unroll
  for (int mp = 0; mp < 2; ++mp) {
    m[mp][0] = m[mp][1] = -INFINITY;
    l[mp][0] = l[mp][1] = 0.f;
#pragma unroll
    for (int n = 0; n < DVT; ++n) o[mp][n][0] = o[mp][n][1] = o[mp][n][2] = o[mp][n][3] = 0.f;
  }
  const DaWalk walk_k = da_walk(2 * d, tid, DA_THREADS), walk_v = da_walk(dv, tid, DA_THREADS);
  auto issue = [&](int n) {               // where[n & 1] holds tile n's cache rows
    const int* list = where[n & 1];
    auto at = [&](int r) { return list[r]; };
    da_load_rows(Ks + (size_t)(n & 1) * DA_KEYS * pitch_k, pitch_k, k_cache, DA_KEYS, walk_k,
                 (DA_KEYS * walk_k.chunks + DA_THREADS - 1) / DA_THREADS, at);
    da_load_rows(Vs + (size_t)(n & 1) * DA_KEYS * pitch_v, pitch_v, v_cache, DA_KEYS, walk_v,
                 (DA_KEYS * walk_v.chunks + DA_THREADS - 1) / DA_THREADS, at);
  };
  auto look_up = [&](int n) {
    if (tid < DA_KEYS)
      where[n & 1][tid] = da_cache_row(table, n * DA_KEYS + tid, p_hi + 1, nkv, g, page_size,
                                       num_pages, err);
  };
  look_up(0);
  __syncthreads();
  issue(0);
  cp_async_commit();
  if (n_tiles > 1) look_up(1);
  __syncthreads();
  for (int n = 0; n < n_tiles; ++n) {
    if (n + 1 < n_tiles) issue(n + 1);    // travels while this one is used
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    if (n + 2 < n_tiles) look_up(n + 2);  // (tile n's list is done with)
    const int base = n * DA_KEYS;
    const __nv_bfloat16* kt = Ks + (size_t)(n & 1) * DA_KEYS * pitch_k;
    const __nv_bfloat16* vt = Vs + (size_t)(n & 1) * DA_KEYS * pitch_v;
    const int rel[2] = {my_p[0] - base, my_p[1] - base};
    const bool whole = base + DA_KEYS - 1 <= wp_lo;
    uint32_t pa[2][DA_KEYS / 16][4];
#pragma unroll
    for (int mp = 0; mp < 2; ++mp)
      da_scores<DA_KEYS>(Qs + (size_t)wrow * pitch_k + mp * d, pitch_k, kt + mp * d, pitch_k, d,
                         lane, rel, whole, sc, m[mp], l[mp], corr[mp], pa[mp]);
    da_values<DA_KEYS, DVT>(vt, pitch_v, dv, lane, pa, corr, o);
    __syncthreads();
  }
  cp_async_wait<0>();
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    float inv[2];
#pragma unroll
    for (int mp = 0; mp < 2; ++mp) {
      float s = l[mp][i];
      s += __shfl_xor_sync(0xffffffffu, s, 1);
      s += __shfl_xor_sync(0xffffffffu, s, 2);
      inv[mp] = s > 0.f ? 1.f / s : 0.f;
    }
    inv[1] *= dd.lambda;
    float ss = 0.f;
#pragma unroll
    for (int n = 0; n < DVT; ++n)
#pragma unroll
      for (int e = 0; e < 2; ++e) {       // (columns beyond dv are zero)
        const float v = o[0][n][2 * i + e] * inv[0] - o[1][n][2 * i + e] * inv[1];
        o[0][n][2 * i + e] = v;
        ss += v * v;
      }
    ss += __shfl_xor_sync(0xffffffffu, ss, 1);
    ss += __shfl_xor_sync(0xffffffffu, ss, 2);
    const int row = row0 + wrow + (lane >> 2) + 8 * i;
    if (row < rows_total) {
      const float f = rsqrtf(ss / (float)dv + dd.eps) * dd.out_factor;
      const int tok = t0 + row / Gh;
      const size_t col0 = (size_t)(g * Gh + row % Gh) * dv + 2 * (lane & 3);
      __nv_bfloat16* dst = out + (size_t)tok * out_stride + col0;
      const __nv_bfloat16* gate =
          dd.gate ? (const __nv_bfloat16*)dd.gate + (size_t)tok * dd.gate_stride + col0 : nullptr;
#pragma unroll
      for (int n = 0; n < DVT; ++n)
        if (n * 8 < dv) {
          float a = o[0][n][2 * i] * f, b = o[0][n][2 * i + 1] * f;
          if (gate) {
            const float2 gv =
                __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gate + n * 8));
            a *= bf_sigmoid_fast(gv.x);
            b *= bf_sigmoid_fast(gv.y);
          }
          *reinterpret_cast<__nv_bfloat162*>(dst + n * 8) = __floats2bfloat162_rn(a, b);
        }
    }
  }
}

// grid (shares / 4, kv heads x blocks of 16 heads, rows)
template <int DVT>
__global__ void __launch_bounds__(DA_THREADS) diff_decode_mma_kernel(
    const __nv_bfloat16* __restrict__ q, long long q_stride,
    const __nv_bfloat16* __restrict__ k_cache, const __nv_bfloat16* __restrict__ v_cache,
    const int* __restrict__ rows, const int* __restrict__ seq_of_token,
    const int* __restrict__ positions, const int* __restrict__ tables, int table_stride,
    float* __restrict__ part_o, float* __restrict__ part_ml, int nh, int nkv, int d, int dv,
    int page_size, int num_pages, int max_splits, float scale_log2, int* __restrict__ err,
    float temp_coef, int temp_every) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __shared__ uint64_t bars[DA_THREADS / 32][DA_DSTAGES];
  bf_pdl_trigger();
  bf_pdl_wait();
  const int Gh = nh / nkv, hblocks = (Gh + 15) / 16;
  const int g = blockIdx.y / hblocks, h0 = (blockIdx.y % hblocks) * 16;
  const int nr = min(16, Gh - h0);
  const int r = blockIdx.z, t = rows ? rows[r] : r;
  const int p = positions[t];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (blockIdx.x == 0 && tid == 0 && p / DA_SHARE >= max_splits) atomicOr(err, BF_ERR_SPLITS);
  if ((int)blockIdx.x * 4 * DA_SHARE > p) return;
  const int pitch_k = 2 * d + 8, pitch_v = dv + 8;
  __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(smem_raw);       // [16][pitch_k]
  constexpr int KT = DA_DKEYS, ST = DA_DSTAGES;
  const size_t per_warp = (size_t)ST * KT * (pitch_k + pitch_v);
  __nv_bfloat16* Ks = Qs + (size_t)16 * pitch_k + warp * per_warp;      // [ST][16][pitch_k]
  __nv_bfloat16* Vs = Ks + (size_t)ST * KT * pitch_k;                   // [ST][16][pitch_v]
  uint64_t* full = bars[warp];
  if (lane == 0) {
    for (int x = 0; x < ST; ++x) bf_mbar_init(full + x, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  const int chunks = 2 * d >> 3;
  for (int i = tid; i < 16 * chunks; i += DA_THREADS) {
    const int hr = i / chunks, c = (i - hr * chunks) << 3;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (hr < nr)
      v = *reinterpret_cast<const uint4*>(q + (size_t)t * q_stride +
                                          (size_t)(g * Gh + h0 + hr) * 2 * d + c);
    *reinterpret_cast<uint4*>(Qs + (size_t)hr * pitch_k + c) = v;
  }
  __syncthreads();
  const int share = blockIdx.x * 4 + warp;
  const int first = share * DA_SHARE;
  if (first > p || share >= max_splits) return;          // (no barrier of the CTA follows)
  const int* table = tables + (size_t)seq_of_token[t] * table_stride;
  const int n_tiles = (min(p, first + DA_SHARE - 1) - first) / KT + 1;
  const float sc0 = scale_log2 * bf_query_temperature(p, temp_coef, temp_every);
  const float sc[2] = {sc0, sc0};
  float m[2][2], l[2][2], corr[2][2];
  float o[2][DVT][4];
#pragma unroll
  for (int mp = 0; mp < 2; ++mp) {
    m[mp][0] = m[mp][1] = -INFINITY;
    l[mp][0] = l[mp][1] = 0.f;
#pragma unroll
    for (int n = 0; n < DVT; ++n) o[mp][n][0] = o[mp][n][1] = o[mp][n][2] = o[mp][n][3] = 0.f;
  }
  // a lane looks a key row up; all lookups of the share are in flight together
  int at[DA_SHARE / 32];
#pragma unroll
  for (int n = 0; n < DA_SHARE / 32; ++n)
    at[n] = da_cache_row(table, first + n * 32 + lane, p + 1, nkv, g, page_size, num_pages, err);
  // keys beyond p (masked, but their values must be finite) take the row of the share's first
  const int safe = max(__shfl_sync(0xffffffffu, at[0], 0), 0);
  auto issue = [&](int n) {               // 16 lanes fetch a key row each, 16 a value row
    int mine = -1;
#pragma unroll
    for (int x = 0; x < DA_SHARE / 32; ++x)
      if (x == n / 2) mine = at[x];
    const int row = lane & 15, st = n % ST;
    int e = __shfl_sync(0xffffffffu, mine, row + (n & 1) * 16);
    if (e < 0) e = safe;
    if (lane == 0) bf_mbar_expect_tx(full + st, (uint32_t)(KT * (2 * d + dv) * 2));
    __syncwarp();
    if (lane < 16)
      bf_bulk_load(Ks + ((size_t)st * KT + row) * pitch_k, k_cache + (size_t)e * 2 * d,
                   (uint32_t)(4 * d), full + st);
    else
      bf_bulk_load(Vs + ((size_t)st * KT + row) * pitch_v, v_cache + (size_t)e * dv,
                   (uint32_t)(2 * dv), full + st);
  };
  for (int n = 0; n < min(ST, n_tiles); ++n) issue(n);
  for (int n = 0; n < n_tiles; ++n) {
    if (!bf_mbar_wait_bounded(full + n % ST, (n / ST) & 1)) {
      atomicOr(err, BF_ERR_WAIT);
      break;
    }
    __syncwarp();
    const __nv_bfloat16* kt = Ks + (size_t)(n % ST) * KT * pitch_k;
    const __nv_bfloat16* vt = Vs + (size_t)(n % ST) * KT * pitch_v;
    const int last = p - (first + n * KT);
    const int rel[2] = {last, last};
    uint32_t pa[2][KT / 16][4];
#pragma unroll
    for (int mp = 0; mp < 2; ++mp)
      da_scores<KT>(Qs + mp * d, pitch_k, kt + mp * d, pitch_k, d, lane, rel,
                    last >= KT - 1, sc, m[mp], l[mp], corr[mp], pa[mp]);
    da_values<KT, DVT>(vt, pitch_v, dv, lane, pa, corr, o);
    __syncwarp();
    if (n + ST < n_tiles) issue(n + ST);
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int hr = (lane >> 2) + 8 * i;
#pragma unroll
    for (int mp = 0; mp < 2; ++mp) {
      float s = l[mp][i];
      s += __shfl_xor_sync(0xffffffffu, s, 1);
      s += __shfl_xor_sync(0xffffffffu, s, 2);
      if (hr < nr) {
        const size_t slot =
            (((size_t)r * nh + g * Gh + h0 + hr) * 2 + mp) * max_splits + share;
        if ((lane & 3) == 0) {
          part_ml[slot * 2] = m[mp][i];
          part_ml[slot * 2 + 1] = s;
        }
#pragma unroll
        for (int n = 0; n < DVT; ++n)
          if (n * 8 < dv)
            *reinterpret_cast<float2*>(part_o + slot * dv + n * 8 + 2 * (lane & 3)) =
                make_float2(o[mp][n][2 * i], o[mp][n][2 * i + 1]);
      }
    }
  }
}

static bool da_takes(int nh, int nkv, int d, int dv, float scale, float temp_coef, int temp_every,
                     const void* q, long long q_stride, const void* k, const void* v) {
  return nkv > 0 && nh % nkv == 0 && d > 0 && dv > 0 && d % 16 == 0 && dv % 16 == 0 && d <= 128 &&
         dv <= 128 && scale > 0.f && temp_coef >= 0.f && temp_every >= 1 && q_stride % 8 == 0 &&
         (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v) & 15) == 0;
}

// The arguments of bf_diff_attention_prefill_umma, with d and dv; no splits.
BF_EXPORT int bf_diff_attention_prefill_mma(
    const void* q, long long q_stride, const void* k_cache, const void* v_cache, const int* items,
    int n_items, int max_rows, const int* block_tables, int table_stride, void* out, int nh,
    int nkv, int d, int dv, int page_size, int num_pages, float scale, int* err,
    long long out_stride, const void* gate, long long gate_stride, float lambda, float eps,
    float out_factor, float temp_coef, int temp_every, cudaStream_t stream) {
  if (n_items <= 0 || max_rows <= 0) return 0;
  if (!da_takes(nh, nkv, d, dv, scale, temp_coef, temp_every, q, q_stride, k_cache, v_cache) ||
      (out_stride & 1) || ((uintptr_t)out & 3) || (gate_stride & 1) || ((uintptr_t)gate & 3))
    return (int)cudaErrorInvalidValue;
  const long long rows = (long long)max_rows * (nh / nkv);
  dim3 grid((unsigned)((rows + DA_ROWS - 1) / DA_ROWS), nkv, n_items);
  if (grid.y > 65535u || grid.z > 65535u) return (int)cudaErrorInvalidValue;
  const size_t smem = (size_t)2 * (DA_ROWS * (2 * d + 8) + 2 * DA_KEYS * (2 * d + 8 + dv + 8));
  auto kern = dv <= 64 ? diff_prefill_mma_kernel<8> : diff_prefill_mma_kernel<16>;
  static bool configured[BF_MAX_DEVICES][2];
  bool& c = configured[bf_current_device()][dv <= 64 ? 0 : 1];
  if (!c) {
    const cudaError_t e =
        cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return (int)e;
    c = true;
  }
  const BfDiffArgs dd = {gate, gate_stride, lambda, eps, out_factor, temp_coef, temp_every};
  kern<<<grid, DA_THREADS, smem, stream>>>(
      (const __nv_bfloat16*)q, q_stride, (const __nv_bfloat16*)k_cache,
      (const __nv_bfloat16*)v_cache, items, block_tables, table_stride, (__nv_bfloat16*)out,
      out_stride, nh, nkv, d, dv, page_size, num_pages, scale * 1.4426950408889634f, err, dd);
  return bf_launch_status();
}

// The arguments of bf_diff_attention_decode_persistent, with d (of one map) and dv.
BF_EXPORT int bf_diff_attention_decode_mma(
    const void* q, long long q_stride, const void* k_cache, const void* v_cache, const int* rows,
    const int* seq_of_token, const int* positions, const int* block_tables, int table_stride,
    void* out, float* part_o, float* part_ml, int n_rows, int nh, int nkv, int d, int dv,
    int page_size, int num_pages, int max_splits, float scale, int* err, long long out_stride,
    const void* gate, long long gate_stride, float lambda, float eps, float out_factor,
    float temp_coef, int temp_every, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (!da_takes(nh, nkv, d, dv, scale, temp_coef, temp_every, q, q_stride, k_cache, v_cache) ||
      max_splits < 1 || !part_o || !part_ml)
    return (int)cudaErrorInvalidValue;
  const int Gh = nh / nkv;
  dim3 grid((max_splits + 3) / 4, nkv * ((Gh + 15) / 16), n_rows);
  if (grid.y > 65535u || grid.z > 65535u) return (int)cudaErrorInvalidValue;
  const size_t smem =
      (size_t)2 * (16 * (2 * d + 8) + 4 * DA_DSTAGES * DA_DKEYS * ((2 * d + 8) + (dv + 8)));
  auto kern = dv <= 64 ? diff_decode_mma_kernel<8> : diff_decode_mma_kernel<16>;
  static bool configured[BF_MAX_DEVICES][2];
  bool& c = configured[bf_current_device()][dv <= 64 ? 0 : 1];
  if (!c) {
    const cudaError_t e =
        cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024);
    if (e != cudaSuccess) return (int)e;
    c = true;
  }
  int e = bf_launch_pdl(kern, grid, dim3(DA_THREADS), smem, stream, (const __nv_bfloat16*)q,
                        q_stride, (const __nv_bfloat16*)k_cache, (const __nv_bfloat16*)v_cache,
                        rows, seq_of_token, positions, block_tables, table_stride, part_o, part_ml,
                        nh, nkv, d, dv, page_size, num_pages, max_splits,
                        scale * 1.4426950408889634f, err, temp_coef, temp_every);
  if (e) return e;
  const BfDiffArgs dd = {gate, gate_stride, lambda, eps, out_factor, temp_coef, temp_every};
  return bf_diff_attention_merge_rows(part_o, part_ml, rows, positions, out, n_rows, nh, dv,
                                      max_splits, out_stride, dd, stream);
}
