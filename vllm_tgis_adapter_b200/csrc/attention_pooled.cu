// Grouped-query softmax attention over a sliding window of tokens plus pooled blocks of the tokens that left it, over a window plus
// the first tokens of the sequence, or inside chunks (kernels.h: PoolAttnGeom).  With a window and pooled blocks, a query at position i sees
//   * the tokens j with 0 <= i - j < window, each with its own key and value, and
//   * every block b of `pool` consecutive positions with b * pool + pool - 1 <= i - window through ONE key and ONE value: the
//     means of the block's cached keys (after rotation and norm) and values,
// all under one softmax.  Tokens behind the window whose block is still incomplete at i - window are not seen at all.  Without
// pooled blocks it may see, beside the window, the tokens j < keep_first; with chunks it sees only tokens of its own chunk.  A sink
// is one more term of the softmax's denominator: the running state (maximum, sum) starts as if one key of that score and of
// weight but without a value had been seen.
//
//   poolattn_prep_kernel   per token and head: bias, rotary turn (fp32 table), unit RMS norm of queries and keys, cache write
//   poolattn_prep_full_kernel  the same with queries and keys normed over all heads at once, values optionally the projected keys
//   poolattn_pool_kernel   the blocks that this step's tokens complete: mean of the block's cache rows -> the pooled cache
//   poolattn_mma_kernel    bf16 rows whose sizes fit the MMA tiles: both products on mma.sync with fp32 accumulators
//   poolattn_kernel        any sizes and fp32 rows (FMA pipe)
//
// The attention kernels take one CTA per (tile of POOLATTN_TILE query tokens of one sequence, query head) and walk "chunks" of
// 32 keys in a fixed order: first the pooled rows 0..31, 32..63, ... that the tile's last query sees, or the cache blocks of the
// first keep_first tokens as far as they lie before the window, then the sequence's 32-token cache blocks from the first one the
// tile's window (or chunk) touches.  Scores, the running softmax (maximum, sum) and the
// accumulators are fp32; a key that a query does not see weighs exactly zero.  So a query row's arithmetic depends on its own
// position and on the 32-row grids of its sequence only: not on the tile it shares with other queries, on how the prompt was cut,
// on the other sequences of the step, or on which physical pages hold the rows.
//
// Pooled rows live in a cache of their own that is paged by the SAME block ids: block b belongs to the page of its first
// token, p = b * pool / KV_BLOCK, at index b - ceil(p * KV_BLOCK / pool); a page owns ceil(KV_BLOCK / pool) of them.
#include <cmath>
#include <cstdint>
#include <algorithm>
#include <cstdlib>
#include <type_traits>

#include "kernels.h"
#include "launch.cuh"
#include "ptx.cuh"

namespace tgis {
namespace {

template <class T>
__device__ __forceinline__ float ldf(const T* p);
template <>
__device__ __forceinline__ float ldf<float>(const float* p) { return *p; }
template <>
__device__ __forceinline__ float ldf<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void stf(float* p, float v) { *p = v; }
__device__ __forceinline__ void stf(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float warp_sum_f(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max_f(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
// pooled blocks a query at position `pos` sees
__device__ __forceinline__ int pooled_visible(int pos, int window, int pool) {
  const int e = pos - window + 1;   // positions [0, e) lie behind the window
  return (window > 0 && pool > 0 && e > 0) ? e / pool : 0;
}
// What a query at position `pos` sees token by token: the keys j <= pos with j >= lo or j < keep
struct Visible { int lo, keep; };
__device__ __forceinline__ Visible visible_tokens(int pos, const PoolAttnGeom& g) {
  const int cl = g.chunk > 0 ? pos / g.chunk * g.chunk : 0;   // first position of the query's chunk
  const int wl = g.window > 0 ? max(0, pos - g.window + 1) : 0;
  return {max(cl, wl), cl > 0 ? 0 : g.keep_first};
}
// factor on the outputs of head h at token row t
__device__ __forceinline__ float out_factor(const PoolAttnGeom& g, int t, int h) {
  return g.head_gate != nullptr ? g.out_mul / (1.f + expf(-g.head_gate[(size_t)t * g.gate_ld + h])) : g.out_mul;
}
__device__ __forceinline__ size_t out_row(const PoolAttnGeom& g, int t) { return (size_t)t * (g.out_ld > 0 ? g.out_ld : g.heads * g.vdim); }
// row of pooled block b inside the pooled cache (page table bt of the sequence)
__device__ __forceinline__ size_t pooled_row(int b, int pool, int rpp, const int32_t* bt) {
  const int page = (int)(((long long)b * pool) / KV_BLOCK);
  const int first = (page * KV_BLOCK + pool - 1) / pool;   // first block whose first token lies in the page
  return (size_t)bt[page] * rpp + (b - first);
}

// ---------------------------------------------------------------------------------------------------------------- prep
// grid (T, ceil((heads + 2 kv_heads) / 4)), 128 threads: one warp per (token, query head | key head | value head)
constexpr int PREP_WARPS = 4, PREP_MAX_DIM = 512;
template <class CT, int PREP_MAX>   // dim <= 32 * PREP_MAX
__global__ void __launch_bounds__(PREP_WARPS * 32)
poolattn_prep_kernel(const float* __restrict__ y, int ldy, int q_off, int k_off, int v_off, const float* __restrict__ bias,
                     PoolAttnGeom g, const float* __restrict__ cos_sin, float eps, const int32_t* __restrict__ positions,
                     const int32_t* __restrict__ slot_mapping, CT* __restrict__ q_out, CT* __restrict__ k_cache,
                     CT* __restrict__ v_cache) {
  griddep_launch();
  griddep_wait();
  const int t = blockIdx.x, hh = blockIdx.y * PREP_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (hh >= g.heads + 2 * g.kv_heads) return;
  const int slot = slot_mapping[t];
  const int nq = g.heads * g.dim, nk = g.kv_heads * g.dim;
  if (hh < g.heads + g.kv_heads) {
    const bool is_q = hh < g.heads;
    const int h = is_q ? hh : hh - g.heads;
    if (!is_q && slot < 0) return;
    const float* src = y + (size_t)t * ldy + (is_q ? q_off : k_off) + (size_t)h * g.dim;
    const float* b = bias != nullptr ? bias + (is_q ? 0 : nq) + (size_t)h * g.dim : nullptr;
    const float* cs = cos_sin != nullptr ? cos_sin + (size_t)positions[t] * g.rot_dims : nullptr;
    const int half = g.rot_dims / 2;
    float val[PREP_MAX];
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < PREP_MAX; ++e) {
      const int i = lane + 32 * e;
      float v = 0.f;
      if (i < g.dim) {
        v = src[i] + (b ? b[i] : 0.f);
        if (i < g.rot_dims) {
          const bool first = g.rot_interleaved ? (i & 1) == 0 : i < half;   // of its pair; the partner is j, the angle's index f
          const int j = g.rot_interleaved ? i ^ 1 : (first ? i + half : i - half), f = g.rot_interleaved ? i >> 1 : (first ? i : j);
          const float w = src[j] + (b ? b[j] : 0.f);
          v = first ? v * cs[f] - w * cs[half + f] : v * cs[f] + w * cs[half + f];
        }
      }
      val[e] = v;
      ss = fmaf(v, v, ss);
    }
    const float rs = g.unit_norm ? 1.f / sqrtf(warp_sum_f(ss) / (float)g.dim + eps) : 1.f;
    CT* dst = is_q ? q_out + ((size_t)t * g.heads + h) * g.dim : k_cache + ((size_t)slot * g.kv_heads + h) * g.dim;
#pragma unroll
    for (int e = 0; e < PREP_MAX; ++e) {
      const int i = lane + 32 * e;
      if (i < g.dim) stf(dst + i, val[e] * rs);
    }
  } else if (slot >= 0) {
    const int h = hh - g.heads - g.kv_heads;
    const float* src = y + (size_t)t * ldy + v_off + (size_t)h * g.vdim;
    const float* b = bias != nullptr ? bias + nq + (v_off == k_off ? 0 : nk) + (size_t)h * g.vdim : nullptr;
    CT* dst = v_cache + ((size_t)slot * g.kv_heads + h) * g.vdim;
    for (int i = lane; i < g.vdim; i += 32) stf(dst + i, src[i] + (b ? b[i] : 0.f));
  }
}

// Queries and keys normed over ALL heads of the token (kernels.h: q_norm / k_norm), optionally with values that are the keys as
// projected: grid (T), 256 threads, one token per CTA.  The row [q | k] (bias added) is staged in shared memory once; its two sums
// of squares are reduced over the CTA, then every pair is normed, turned and stored.
constexpr int PREPF_THREADS = 256;
template <class CT>
__global__ void __launch_bounds__(PREPF_THREADS)
poolattn_prep_full_kernel(const float* __restrict__ y, int ldy, int q_off, int k_off, int v_off, const float* __restrict__ bias,
                          PoolAttnGeom g, const float* __restrict__ cos_sin, float eps, const int32_t* __restrict__ positions,
                          const int32_t* __restrict__ slot_mapping, CT* __restrict__ q_out, CT* __restrict__ k_cache,
                          CT* __restrict__ v_cache) {
  extern __shared__ float prow[];   // [heads * dim | kv_heads * dim]
  __shared__ float red[2][PREPF_THREADS / 32];
  griddep_launch();
  griddep_wait();
  const int t = blockIdx.x, tid = threadIdx.x, slot = slot_mapping[t];
  const int nq = g.heads * g.dim, nk = g.kv_heads * g.dim, nv = g.kv_heads * g.vdim;
  const float* src = y + (size_t)t * ldy;
  const bool shared_kv = v_off == k_off;
  float sq = 0.f, sk = 0.f;
  for (int i = tid; i < nq + nk; i += PREPF_THREADS) {
    const bool is_q = i < nq;
    const float v = src[is_q ? q_off + i : k_off + i - nq] + (bias != nullptr ? bias[i] : 0.f);
    prow[i] = v;
    if (is_q) sq = fmaf(v, v, sq);
    else sk = fmaf(v, v, sk);
  }
  sq = warp_sum_f(sq);
  sk = warp_sum_f(sk);
  if ((tid & 31) == 0) {
    red[0][tid >> 5] = sq;
    red[1][tid >> 5] = sk;
  }
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int w = 0; w < PREPF_THREADS / 32; ++w) {   // the same order in every thread
    sq += red[0][w];
    sk += red[1][w];
  }
  const float rq = 1.f / sqrtf(sq / (float)nq + eps), rk = 1.f / sqrtf(sk / (float)nk + eps);
  const float* cs = cos_sin != nullptr ? cos_sin + (size_t)positions[t] * g.rot_dims : nullptr;
  const int half = g.rot_dims / 2;
  for (int i = tid; i < nq + nk; i += PREPF_THREADS) {
    const bool is_q = i < nq;
    if (!is_q && slot < 0) break;
    const float* w = is_q ? g.q_norm : g.k_norm - nq;
    const float rs = is_q ? rq : rk;
    const int d = (is_q ? i : i - nq) % g.dim;
    float v = prow[i] * rs * w[i];
    if (d < g.rot_dims) {
      const bool first = g.rot_interleaved ? (d & 1) == 0 : d < half;
      const int j = i + (g.rot_interleaved ? (first ? 1 : -1) : (first ? half : -half));
      const int f = g.rot_interleaved ? d >> 1 : (first ? d : d - half);
      const float p = prow[j] * rs * w[j];
      v = first ? v * cs[f] - p * cs[half + f] : v * cs[f] + p * cs[half + f];
    }
    if (is_q) stf(q_out + (size_t)t * nq + i, v);
    else stf(k_cache + (size_t)slot * nk + i - nq, v);
  }
  if (slot >= 0) {
    for (int i = tid; i < nv; i += PREPF_THREADS)
      stf(v_cache + (size_t)slot * nv + i, shared_kv ? prow[nq + i] : src[v_off + i] + (bias != nullptr ? bias[nq + nk + i] : 0.f));
  }
}

// poolattn_prep_full_kernel for interleaved pairs (or none) with shared keys and values, sizes that are multiples of four and rows
// on 16-byte boundaries: two pairs per thread and step, kept in registers between the passes
constexpr int PREPF_V = 4;   // (heads + kv_heads) * dim <= 4 PREPF_THREADS PREPF_V
template <class CT>
__device__ __forceinline__ void st4(CT* p, float4 v);
template <>
__device__ __forceinline__ void st4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <>
__device__ __forceinline__ void st4<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  uint2 pk;
  pk.x = *reinterpret_cast<const uint32_t*>(&lo);
  pk.y = *reinterpret_cast<const uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(p) = pk;
}
template <class CT>
__global__ void __launch_bounds__(PREPF_THREADS)
poolattn_prep_full_vec_kernel(const float* __restrict__ y, int ldy, int q_off, int k_off, const float* __restrict__ bias, PoolAttnGeom g,
                              const float* __restrict__ cos_sin, float eps, const int32_t* __restrict__ positions,
                              const int32_t* __restrict__ slot_mapping, CT* __restrict__ q_out, CT* __restrict__ k_cache,
                              CT* __restrict__ v_cache) {
  __shared__ float red[2][PREPF_THREADS / 32];
  griddep_launch();
  griddep_wait();
  const int t = blockIdx.x, tid = threadIdx.x, slot = slot_mapping[t];
  const int nq = g.heads * g.dim, nk = g.kv_heads * g.dim;
  const float* src = y + (size_t)t * ldy;
  float4 v[PREPF_V];
  float sq = 0.f, sk = 0.f;
#pragma unroll
  for (int e = 0; e < PREPF_V; ++e) {
    const int i = (e * PREPF_THREADS + tid) * 4;
    v[e] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < nq + nk) {
      v[e] = *reinterpret_cast<const float4*>(src + (i < nq ? q_off + i : k_off + i - nq));
      if (bias != nullptr) {
        const float4 b = *reinterpret_cast<const float4*>(bias + i);
        v[e].x += b.x; v[e].y += b.y; v[e].z += b.z; v[e].w += b.w;
      }
    }
    const float s = fmaf(v[e].x, v[e].x, fmaf(v[e].y, v[e].y, fmaf(v[e].z, v[e].z, v[e].w * v[e].w)));
    if (i < nq) sq += s;
    else sk += s;
  }
  sq = warp_sum_f(sq);
  sk = warp_sum_f(sk);
  if ((tid & 31) == 0) {
    red[0][tid >> 5] = sq;
    red[1][tid >> 5] = sk;
  }
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int w = 0; w < PREPF_THREADS / 32; ++w) {   // the same order in every thread
    sq += red[0][w];
    sk += red[1][w];
  }
  const float rq = 1.f / sqrtf(sq / (float)nq + eps), rk = 1.f / sqrtf(sk / (float)nk + eps);
  const float* cs = cos_sin != nullptr ? cos_sin + (size_t)positions[t] * g.rot_dims : nullptr;
  const int half = g.rot_dims / 2;
#pragma unroll
  for (int e = 0; e < PREPF_V; ++e) {
    const int i = (e * PREPF_THREADS + tid) * 4;
    const bool is_q = i < nq;
    if (i >= nq + nk || (!is_q && slot < 0)) break;
    const float4 w = *reinterpret_cast<const float4*>(is_q ? g.q_norm + i : g.k_norm + i - nq);
    const float rs = is_q ? rq : rk;
    const int d = (is_q ? i : i - nq) % g.dim;
    float4 x = make_float4(v[e].x * rs * w.x, v[e].y * rs * w.y, v[e].z * rs * w.z, v[e].w * rs * w.w);
    if (d < g.rot_dims) {
      const float2 c = *reinterpret_cast<const float2*>(cs + d / 2), s = *reinterpret_cast<const float2*>(cs + half + d / 2);
      x = make_float4(x.x * c.x - x.y * s.x, x.y * c.x + x.x * s.x, x.z * c.y - x.w * s.y, x.w * c.y + x.z * s.y);
    }
    if (is_q) {
      st4(q_out + (size_t)t * nq + i, x);
    } else {
      st4(k_cache + (size_t)slot * nk + i - nq, x);
      st4(v_cache + (size_t)slot * nk + i - nq, v[e]);
    }
  }
}

// ---------------------------------------------------------------------------------------------------------------- pool
// grid (sequences, blocks per sequence in strides of gridDim.y), 128 threads over the columns of a K | V row
template <class CT>
__global__ void __launch_bounds__(128)
poolattn_pool_kernel(const CT* __restrict__ k_cache, const CT* __restrict__ v_cache, CT* __restrict__ pk, CT* __restrict__ pv,
                     const AttnSeq* __restrict__ seqs, const int32_t* __restrict__ block_table, int bt_stride, PoolAttnGeom g) {
  griddep_launch();
  griddep_wait();
  const AttnSeq sq = seqs[blockIdx.x];
  const int P = g.pool, first = sq.kv_len - sq.q_len;
  const int b_lo = first / P, b_hi = sq.kv_len / P;   // blocks whose last position is one of this step's tokens
  const int32_t* bt = block_table + (size_t)sq.block_row * bt_stride;
  const int nk = g.kv_heads * g.dim, nv = g.kv_heads * g.vdim, rpp = g.rows_per_page();
  const float inv = 1.f / (float)P;
  for (int b = b_lo + blockIdx.y; b < b_hi; b += gridDim.y) {
    const size_t dst = pooled_row(b, P, rpp, bt);
    if (sizeof(CT) == 2 && nk % 8 == 0 && nv % 8 == 0) {   // bf16 rows of whole 16-byte groups: eight columns per thread
      for (int c8 = threadIdx.x; c8 < (nk + nv) / 8; c8 += blockDim.x) {
        const bool is_k = c8 < nk / 8;
        const int col = is_k ? c8 * 8 : c8 * 8 - nk;
        float s8[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
        for (int r = 0; r < P; ++r) {   // position order
          const int pos = b * P + r;
          const size_t row = (size_t)bt[pos / KV_BLOCK] * KV_BLOCK + pos % KV_BLOCK;
          const uint4 v = *reinterpret_cast<const uint4*>(is_k ? reinterpret_cast<const __nv_bfloat16*>(k_cache) + row * nk + col
                                                               : reinterpret_cast<const __nv_bfloat16*>(v_cache) + row * nv + col);
          const __nv_bfloat162* v2 = reinterpret_cast<const __nv_bfloat162*>(&v);
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            s8[2 * e] += __bfloat162float(v2[e].x);
            s8[2 * e + 1] += __bfloat162float(v2[e].y);
          }
        }
        uint4 o;
        __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
        for (int e = 0; e < 4; ++e) o2[e] = __floats2bfloat162_rn(s8[2 * e] * inv, s8[2 * e + 1] * inv);
        *reinterpret_cast<uint4*>(is_k ? reinterpret_cast<__nv_bfloat16*>(pk) + dst * nk + col
                                       : reinterpret_cast<__nv_bfloat16*>(pv) + dst * nv + col) = o;
      }
      continue;
    }
    for (int c = threadIdx.x; c < nk + nv; c += blockDim.x) {
      float s = 0.f;
#pragma unroll 4
      for (int r = 0; r < P; ++r) {   // position order
        const int pos = b * P + r;
        const size_t row = (size_t)bt[pos / KV_BLOCK] * KV_BLOCK + pos % KV_BLOCK;
        s += c < nk ? ldf(k_cache + row * nk + c) : ldf(v_cache + row * nv + (c - nk));
      }
      if (c < nk) stf(pk + dst * nk + c, s * inv);
      else stf(pv + dst * nv + (c - nk), s * inv);
    }
  }
}

// ---------------------------------------------------------------------------------------------------------------- FMA kernel
constexpr int PA_THREADS = 128, PA_QT = POOLATTN_TILE, PA_CC = POOLATTN_MAX_VDIM / PA_THREADS;
static_assert(PA_QT == 16 && PA_THREADS == 128, "score mapping: 4 warps x 4 queries x 32 keys");

template <class CT, class OT>
__global__ void __launch_bounds__(PA_THREADS)
poolattn_kernel(const CT* __restrict__ q, const CT* __restrict__ k_cache, const CT* __restrict__ v_cache,
                const CT* __restrict__ pk, const CT* __restrict__ pv, const AttnSeq* __restrict__ seqs,
                const LatentTile* __restrict__ tiles, const int32_t* __restrict__ block_table, int bt_stride,
                OT* __restrict__ out, PoolAttnGeom g) {
  extern __shared__ __align__(16) float pa_smem[];
  const int d = g.dim, dv = g.vdim, ldk = d + 1;
  float* Qs = pa_smem;                        // [PA_QT][d]      scaled queries
  float* Ks = Qs + PA_QT * d;                 // [KV_BLOCK][d+1]
  float* Vs = Ks + KV_BLOCK * ldk;            // [KV_BLOCK][dv]
  float* Ps = Vs + KV_BLOCK * dv;             // [PA_QT][KV_BLOCK]
  float* alpha = Ps + PA_QT * KV_BLOCK;       // [PA_QT]
  float* lsum = alpha + PA_QT;                // [PA_QT]
  __shared__ long long rowoff[KV_BLOCK];      // cache row of every key of the chunk (-1: none)
  __shared__ float fac[PA_QT];                // factors of the tile's outputs
  griddep_launch();
  griddep_wait();
  const LatentTile tl = tiles[blockIdx.x];
  const AttnSeq sq = seqs[tl.seq];
  const int h = blockIdx.y, kvh = h / (g.heads / g.kv_heads);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int row0 = sq.q_start + tl.q0;             // first query row of the tile in the flat batch
  const int pos0 = sq.kv_len - sq.q_len + tl.q0;   // its position
  const int nq = tl.nq, pos_last = pos0 + nq - 1;
  for (int i = tid; i < PA_QT * d; i += PA_THREADS) {
    const int qi = i / d, kk = i % d;
    Qs[i] = qi < nq ? ldf(q + ((size_t)(row0 + qi) * g.heads + h) * d + kk) * g.scale : 0.f;
  }
  float acc[PA_QT][PA_CC];
#pragma unroll
  for (int qi = 0; qi < PA_QT; ++qi)
#pragma unroll
    for (int cc = 0; cc < PA_CC; ++cc) acc[qi][cc] = 0.f;
  float m_run[4], l_run[4];   // this warp's four query rows (valid in every lane)
  int n_vis[4];               // pooled blocks each of them sees
  Visible vis[4];             // ... and tokens
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    m_run[i] = g.sink != nullptr ? g.sink[h] : -INFINITY;
    l_run[i] = g.sink != nullptr ? 1.f : 0.f;
    vis[i] = visible_tokens(pos0 + warp * 4 + i, g);
    n_vis[i] = pooled_visible(pos0 + warp * 4 + i, g.window, g.pool);
  }
  const int n_pooled = pooled_visible(pos_last, g.window, g.pool);
  const Visible first = visible_tokens(pos0, g);
  const int blk0 = first.lo / KV_BLOCK, blk1 = pos_last / KV_BLOCK;
  // chunks in front of the window's blocks: pooled rows, or the blocks of the kept first tokens
  const int n_pc = g.pool > 0 ? (n_pooled + KV_BLOCK - 1) / KV_BLOCK : min((first.keep + KV_BLOCK - 1) / KV_BLOCK, blk0);
  const int n_chunks = n_pc + blk1 - blk0 + 1;
  const int rpp = g.rows_per_page();
  const int32_t* bt = block_table + (size_t)sq.block_row * bt_stride;
  for (int c = 0; c < n_chunks; ++c) {
    const bool pooled = g.pool > 0 && c < n_pc;
    const int blk = c < n_pc ? c : blk0 + c - n_pc;   // pooled chunk, or cache block of the sequence
    __syncthreads();   // the previous chunk's Ks / Vs / Ps / rowoff are consumed (first pass: Qs complete)
    if (tid < KV_BLOCK) {
      long long r;
      if (pooled) {
        const int b = blk * KV_BLOCK + tid;
        r = b < n_pooled ? (long long)pooled_row(b, g.pool, rpp, bt) : -1;
      } else {
        r = (long long)bt[blk] * KV_BLOCK + tid;
      }
      rowoff[tid] = r;
    }
    __syncthreads();
    const CT* kb = pooled ? pk : k_cache;
    const CT* vb = pooled ? pv : v_cache;
    for (int i = tid; i < KV_BLOCK * d; i += PA_THREADS) {
      const int j = i / d, kk = i % d;
      const long long r = rowoff[j];
      Ks[j * ldk + kk] = r >= 0 ? ldf(kb + ((size_t)r * g.kv_heads + kvh) * d + kk) : 0.f;
    }
    for (int i = tid; i < KV_BLOCK * dv; i += PA_THREADS) {
      const int j = i / dv, cc = i % dv;
      const long long r = rowoff[j];
      Vs[i] = r >= 0 ? ldf(vb + ((size_t)r * g.kv_heads + kvh) * dv + cc) : 0.f;
    }
    __syncthreads();
    // ---- scores: lane = key, this warp's four queries
    float s[4] = {0.f, 0.f, 0.f, 0.f};
    const float* kr = Ks + lane * ldk;
    const float* qr = Qs + warp * 4 * d;
    for (int kk = 0; kk < d; ++kk) {
      const float kv = kr[kk];
#pragma unroll
      for (int i = 0; i < 4; ++i) s[i] = fmaf(qr[i * d + kk], kv, s[i]);
    }
    const int kidx = blk * KV_BLOCK + lane;   // pooled block number, or token position
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int qi = warp * 4 + i, pi = pos0 + qi;
      const bool ok = qi < nq && (pooled ? kidx < n_vis[i] : (kidx <= pi && (kidx >= vis[i].lo || kidx < vis[i].keep)));
      const float sc = ok ? s[i] : -INFINITY;
      const float m_new = fmaxf(m_run[i], warp_max_f(sc));
      const float p = ok ? expf(sc - m_new) : 0.f;
      const float al = m_new == -INFINITY ? 1.f : expf(m_run[i] - m_new);   // (-inf: nothing seen yet, nothing to scale)
      l_run[i] = fmaf(l_run[i], al, warp_sum_f(p));
      m_run[i] = m_new;
      Ps[qi * KV_BLOCK + lane] = p;
      if (lane == 0) alpha[qi] = al;
    }
    __syncthreads();
    // ---- weighted sum of the values: thread = value column(s), all queries of the tile
#pragma unroll
    for (int cc = 0; cc < PA_CC; ++cc) {
      const int col = tid + cc * PA_THREADS;
      if (col < dv) {
#pragma unroll
        for (int qi = 0; qi < PA_QT; ++qi)
          if (qi < nq) acc[qi][cc] *= alpha[qi];
        for (int j = 0; j < KV_BLOCK; ++j) {
          const float vv = Vs[j * dv + col];
#pragma unroll
          for (int qi = 0; qi < PA_QT; ++qi)
            if (qi < nq) acc[qi][cc] = fmaf(Ps[qi * KV_BLOCK + j], vv, acc[qi][cc]);
        }
      }
    }
  }
  if (lane == 0) {
#pragma unroll
    for (int i = 0; i < 4; ++i) lsum[warp * 4 + i] = l_run[i];
  }
  if (tid < nq) fac[tid] = out_factor(g, row0 + tid, h);
  __syncthreads();
#pragma unroll
  for (int cc = 0; cc < PA_CC; ++cc) {
    const int col = tid + cc * PA_THREADS;
    if (col < dv) {
#pragma unroll
      for (int qi = 0; qi < PA_QT; ++qi)
        if (qi < nq) stf(out + out_row(g, row0 + qi) + (size_t)h * dv + col, acc[qi][cc] * (fac[qi] / lsum[qi]));
    }
  }
}

// ---------------------------------------------------------------------------------------------------------------- tensor cores
// bf16 queries and cache rows, dim a multiple of 16 (<= 16 MMA_KS), vdim a multiple of 8 (<= 8 NT).  Both products on mma.sync
// m16n8k16 with fp32 accumulators.  A warp owns 16 rows -- (token, query head) pairs of ONE key/value head -- from their scores to
// their outputs: the query's A fragments stay in registers for the whole walk, a chunk's 32 scores per row, the running maximum and
// sum and the accumulators never leave the warp, and the softmax weights become the A fragments of the second product as they lie.
// Scale, mask and the running softmax are fp32 on the accumulator fragments; the weights are rounded to bf16 once and the SAME
// rounded numbers are summed for the normaliser.  Pooled chunks and token chunks differ only in where a row comes from and in
// which queries see it; a warp passes over a chunk that none of its rows sees.
//
// Two shapes of the same walk, four warps each; chunks arrive in a ring through 16-byte asynchronous copies:
//   SPLIT = false  64 rows per CTA, 16 per warp: a chunk's rows are fetched once for all four warps (prompts and portions)
//   SPLIT = true   16 rows per CTA, and every warp walks every fourth chunk on its own, without any CTA-wide barrier; the four
//                  (maximum, sum, accumulator) states meet once at the end (decoded tokens: few rows, long walks)
constexpr int MMA_KS = 8, MMA_MAX_NT = 32;
template <bool SPLIT>
struct PaShape {
  static constexpr int ROWS = SPLIT ? 16 : 64, CPS = SPLIT ? 4 : 1, NST = SPLIT ? 2 : 4;   // rows per CTA, chunks per ring stage, stages
};
__device__ __forceinline__ void pa_ldsm_x4(uint32_t (&r)[4], const void* smem) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(smem);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void pa_ldsm_x4_trans(uint32_t (&r)[4], const void* smem) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(smem);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void pa_cp_async16(void* smem, const void* gmem) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(a), "l"(gmem) : "memory");
}
__device__ __forceinline__ void pa_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// 2^x of the special function unit (relative error of a few 2^-23; results below 2^-126 become zero)
__device__ __forceinline__ float pa_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// KS > 0: the sizes are compile-time constants, dim = 16 KS and vdim = 8 NT; KS = 0: any sizes with dim <= 16 MMA_KS, vdim <= 8 NT
template <int KS, int NT, bool SPLIT>
__global__ void __launch_bounds__(PA_THREADS, !SPLIT && NT <= 16 ? 3 : 1)
poolattn_mma_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ k_cache,
                    const __nv_bfloat16* __restrict__ v_cache, const __nv_bfloat16* __restrict__ pk,
                    const __nv_bfloat16* __restrict__ pv, const AttnSeq* __restrict__ seqs, const LatentTile* __restrict__ tiles,
                    const int32_t* __restrict__ block_table, int bt_stride, __nv_bfloat16* __restrict__ out, PoolAttnGeom g, int gs) {
  // gs: query heads of a key/value head that share a CTA's rows (1, 2, 4, 8 or 16).  Row r: token r / gs of the CTA's ROWS / gs,
  // head h_base + r % gs.  Grid (tiles, heads / gs, max(1, 16 gs / ROWS)): CTA z takes every ROWS / gs tokens of a 16-token tile; where
  // a CTA takes more than a tile's 16 tokens, the tiles in between have nothing to do.
  using bf = __nv_bfloat16;
  using SH = PaShape<SPLIT>;
  extern __shared__ __align__(16) uint8_t pam_smem[];
  constexpr int KSM = KS > 0 ? KS : MMA_KS;
  constexpr bool EXACT = KS > 0;
  const int d = EXACT ? 16 * KS : g.dim, dv = EXACT ? 8 * NT : g.vdim, LDK = d + 8, LDV = dv + 8;
  bf* Ks2 = reinterpret_cast<bf*>(pam_smem);                     // [NST * CPS][32][LDK]   (first the queries: [ROWS][LDK])
  bf* Vs2 = Ks2 + (size_t)SH::NST * SH::CPS * KV_BLOCK * LDK;    // [NST * CPS][32][LDV]
  griddep_launch();
  griddep_wait();
  const LatentTile tl = tiles[blockIdx.x];
  const AttnSeq sq = seqs[tl.seq];
  const int tpt = SH::ROWS / gs;   // tokens per CTA
  int tok0 = tl.q0, nq;
  if (tpt > PA_QT) {
    if (tl.q0 % tpt != 0) return;
    nq = min(tpt, sq.q_len - tok0);
  } else {
    const int off = blockIdx.z * tpt;
    if (off >= tl.nq) return;
    tok0 += off;
    nq = min(tpt, tl.nq - off);
  }
  const int h_base = blockIdx.y * gs, kvh = h_base / (g.heads / g.kv_heads);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, t2 = (lane & 3) * 2;
  const int row0 = sq.q_start + tok0, pos0 = sq.kv_len - sq.q_len + tok0, pos_last = pos0 + nq - 1;
  const int dch = d / 8, vch = dv / 8;   // 16-byte pieces per row
  for (int i = tid; i < SH::ROWS * dch; i += PA_THREADS) {
    const int r = i / dch, ch = i % dch, tq = r / gs;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (tq < nq) v = *reinterpret_cast<const uint4*>(q + ((size_t)(row0 + tq) * g.heads + h_base + r % gs) * d + ch * 8);
    *reinterpret_cast<uint4*>(Ks2 + r * LDK + ch * 8) = v;
  }
  __syncthreads();
  const int nks = d / 16, wr0 = SPLIT ? 0 : warp * 16;   // the warp's first row
  uint32_t qa[KSM][4];
#pragma unroll
  for (int ks = 0; ks < KSM; ++ks)
    if (EXACT || ks < nks) pa_ldsm_x4(qa[ks], Ks2 + (size_t)(wr0 + (lane & 15)) * LDK + ks * 16 + (lane >> 4) * 8);
  __syncthreads();   // the ring may overwrite the queries
  float acc[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
  // scores and maxima in units of ln 2: weights are powers of two
  constexpr float LOG2E = 1.4426950408889634f;
  const float scale2 = g.scale * LOG2E;
  float m_run[2] = {-INFINITY, -INFINITY}, l_part[2] = {0.f, 0.f};   // rows gq and gq + 8 of the warp
  if (g.sink != nullptr) {
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      m_run[r] = g.sink[h_base + (wr0 + gq + r * 8) % gs] * LOG2E;
      l_part[r] = ((!SPLIT || warp == 0) && (lane & 3) == 0) ? 1.f : 0.f;   // (the row's sum adds up the parts of all its threads)
    }
  }
  const int tqr[2] = {(wr0 + gq) / gs, (wr0 + gq + 8) / gs};   // tokens of this thread's two rows
  const Visible vis[2] = {visible_tokens(pos0 + tqr[0], g), visible_tokens(pos0 + tqr[1], g)};
  const int n_vis[2] = {pooled_visible(pos0 + tqr[0], g.window, g.pool), pooled_visible(pos0 + tqr[1], g.window, g.pool)};
  // the warp's first and last token: which chunks concern it at all
  const int tq_lo = wr0 / gs, tq_hi = min((wr0 + 15) / gs, nq - 1);
  const Visible w_first = visible_tokens(pos0 + tq_lo, g), w_last = visible_tokens(pos0 + tq_hi, g);
  const int w_pooled = pooled_visible(pos0 + tq_hi, g.window, g.pool), w_pooled_all = pooled_visible(pos0 + tq_lo, g.window, g.pool);
  const bool w_rows_all = (wr0 + 15) / gs < nq;
  const int n_pooled = pooled_visible(pos_last, g.window, g.pool);
  const Visible first = visible_tokens(pos0, g);
  const int blk0 = first.lo / KV_BLOCK, blk1 = pos_last / KV_BLOCK;
  // chunks in front of the window's blocks: pooled rows, or the blocks of the kept first tokens
  const int n_pc = g.pool > 0 ? (n_pooled + KV_BLOCK - 1) / KV_BLOCK : min((first.keep + KV_BLOCK - 1) / KV_BLOCK, blk0);
  const int n_chunks = n_pc + blk1 - blk0 + 1, n_it = (n_chunks + SH::CPS - 1) / SH::CPS;
  const int rpp = g.rows_per_page();
  const int32_t* bt = block_table + (size_t)sq.block_row * bt_stride;
  // one row of chunk c -> row fj of ring buffer `buf`, four threads per row; pooled rows that do not exist yet are zeros
  auto fetch_row = [&](int c, int buf, int fj, int fl) {
    const bool pooled = g.pool > 0 && c < n_pc;
    const int blk = c < n_pc ? c : blk0 + c - n_pc;   // pooled chunk, or cache block of the sequence
    long long r;
    if (pooled) {
      const int b = blk * KV_BLOCK + fj;
      r = b < n_pooled ? (long long)pooled_row(b, g.pool, rpp, bt) : -1;
    } else {
      r = (long long)__ldg(bt + blk) * KV_BLOCK + fj;
    }
    bf* Kd = Ks2 + ((size_t)buf * KV_BLOCK + fj) * LDK;
    bf* Vd = Vs2 + ((size_t)buf * KV_BLOCK + fj) * LDV;
    if (r < 0) {
      for (int ch = fl; ch < dch; ch += 4) *reinterpret_cast<uint4*>(Kd + ch * 8) = make_uint4(0, 0, 0, 0);
      for (int ch = fl; ch < vch; ch += 4) *reinterpret_cast<uint4*>(Vd + ch * 8) = make_uint4(0, 0, 0, 0);
    } else {
      const bf* ks = (pooled ? pk : k_cache) + ((size_t)r * g.kv_heads + kvh) * d;
      const bf* vs = (pooled ? pv : v_cache) + ((size_t)r * g.kv_heads + kvh) * dv;
      for (int ch = fl; ch < dch; ch += 4) pa_cp_async16(Kd + ch * 8, ks + ch * 8);
      for (int ch = fl; ch < vch; ch += 4) pa_cp_async16(Vd + ch * 8, vs + ch * 8);
    }
  };
  // every call is one commit group (an empty one past the last chunk), so that the group count tells which chunk has landed
  auto fetch = [&](int it) {
    if (SPLIT) {   // the warp's own chunk of the stage
      const int c = it * SH::CPS + warp;
      if (c < n_chunks)
        for (int p = 0; p < 4; ++p) fetch_row(c, (it % SH::NST) * SH::CPS + warp, p * 8 + (lane >> 2), lane & 3);
    } else if (it < n_chunks) {
      fetch_row(it, it % SH::NST, tid >> 2, tid & 3);
    }
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
#pragma unroll
  for (int it = 0; it < SH::NST - 1; ++it) fetch(it);
  for (int it = 0; it < n_it; ++it) {
    asm volatile("cp.async.wait_group %0;\n" ::"n"(SH::NST - 2) : "memory");
    // this pass's chunk has landed for every thread that reads it, and the stage fetched into next is consumed
    if (SPLIT) __syncwarp();
    else __syncthreads();
    fetch(it + SH::NST - 1);
    const int c = SPLIT ? it * SH::CPS + warp : it, buf = SPLIT ? (it % SH::NST) * SH::CPS + warp : it % SH::NST;
    const bool pooled = g.pool > 0 && c < n_pc;
    const int blk = c < n_pc ? c : blk0 + c - n_pc, key0 = blk * KV_BLOCK;   // first pooled block number, or token position
    const bool idle = c >= n_chunks || tq_lo >= nq ||
                      (pooled ? key0 >= w_pooled : key0 > pos0 + tq_hi || (key0 + KV_BLOCK <= w_first.lo && key0 >= w_first.keep));
    if (!idle) {   // (the same for the whole warp)
      const bf* Ks = Ks2 + (size_t)buf * KV_BLOCK * LDK;
      const bf* Vs = Vs2 + (size_t)buf * KV_BLOCK * LDV;
      float sc[4][4];   // keys 8 j + t2, 8 j + t2 + 1 of rows gq and gq + 8
#pragma unroll
      for (int j = 0; j < 4; ++j) sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < KSM; ++ks)
        if (EXACT || ks < nks) {
#pragma unroll
          for (int jj = 0; jj < 2; ++jj) {
            uint32_t kb[4];
            pa_ldsm_x4(kb, Ks + (size_t)(jj * 16 + (lane >> 4) * 8 + (lane & 7)) * LDK + ks * 16 + ((lane >> 3) & 1) * 8);
            pa_mma(sc[2 * jj], qa[ks], kb[0], kb[1]);
            pa_mma(sc[2 * jj + 1], qa[ks], kb[2], kb[3]);
          }
        }
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[j][e] *= scale2;
      // a chunk that every row of the warp sees whole needs no mask
      const bool whole = w_rows_all && (pooled ? key0 + KV_BLOCK <= w_pooled_all
                                               : key0 + KV_BLOCK - 1 <= pos0 + tq_lo && (key0 >= w_last.lo || key0 + KV_BLOCK <= w_last.keep));
      if (!whole) {
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int pi = tqr[r] < nq ? pos0 + tqr[r] : -1;
#pragma unroll
          for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              const int kidx = key0 + j * 8 + t2 + e;
              const bool ok = pooled ? (pi >= 0 && kidx < n_vis[r]) : (kidx <= pi && (kidx >= vis[r].lo || kidx < vis[r].keep));
              if (!ok) sc[j][2 * r + e] = -INFINITY;
            }
        }
      }
      float al[2];
      uint32_t pa[2][4];   // the weights as A fragments of the two 16-key steps of the second product
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        float mx = fmaxf(fmaxf(fmaxf(sc[0][2 * r], sc[0][2 * r + 1]), fmaxf(sc[1][2 * r], sc[1][2 * r + 1])),
                         fmaxf(fmaxf(sc[2][2 * r], sc[2][2 * r + 1]), fmaxf(sc[3][2 * r], sc[3][2 * r + 1])));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float m_new = fmaxf(m_run[r], mx), m_ref = m_new == -INFINITY ? 0.f : m_new;   // (-inf: nothing seen yet)
        al[r] = m_new == -INFINITY ? 1.f : pa_exp2(m_run[r] - m_new);
        float sum = 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) {   // exactly zero for a key that is not seen
          const __nv_bfloat162 pp = __floats2bfloat162_rn(pa_exp2(sc[j][2 * r] - m_ref), pa_exp2(sc[j][2 * r + 1] - m_ref));
          const float2 pf = __bfloat1622float2(pp);
          sum += pf.x + pf.y;
          pa[j >> 1][(j & 1) * 2 + r] = *reinterpret_cast<const uint32_t*>(&pp);
        }
        l_part[r] = fmaf(l_part[r], al[r], sum);
        m_run[r] = m_new;
      }
      if (__any_sync(0xffffffffu, al[0] != 1.f || al[1] != 1.f)) {   // some row's maximum moved
#pragma unroll
        for (int j = 0; j < NT; ++j) { acc[j][0] *= al[0]; acc[j][1] *= al[0]; acc[j][2] *= al[1]; acc[j][3] *= al[1]; }
      }
#pragma unroll
      for (int j = 0; j < NT; ++j)
        if (EXACT || j * 8 < dv) {
          uint32_t vb[4];
          pa_ldsm_x4_trans(vb, Vs + (size_t)lane * LDV + j * 8);
          pa_mma(acc[j], pa[0], vb[0], vb[1]);
          pa_mma(acc[j], pa[1], vb[2], vb[3]);
        }
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l_part[r] += __shfl_xor_sync(0xffffffffu, l_part[r], 1);
    l_part[r] += __shfl_xor_sync(0xffffffffu, l_part[r], 2);
  }
  if (!SPLIT) {
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      if (tqr[r] >= nq) continue;
      const int h = h_base + (wr0 + gq + r * 8) % gs;
      const float inv_l = out_factor(g, row0 + tqr[r], h) / l_part[r];
      bf* dst = out + out_row(g, row0 + tqr[r]) + (size_t)h * dv + t2;
#pragma unroll
      for (int j = 0; j < NT; ++j)
        if (EXACT || j * 8 < dv) *reinterpret_cast<__nv_bfloat162*>(dst + j * 8) = __floats2bfloat162_rn(acc[j][2 * r] * inv_l, acc[j][2 * r + 1] * inv_l);
    }
    return;
  }
  // ---- the four warps' states of the same rows meet, in warp order
  __syncthreads();   // the ring is consumed
  float* ms = reinterpret_cast<float*>(pam_smem);   // [4][16] maxima, [4][16] sums, [4][16][dv] accumulators
  float* ls = ms + 4 * 16;
  float* as = ls + 4 * 16;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int row = gq + r * 8;
    if ((lane & 3) == 0) {
      ms[warp * 16 + row] = m_run[r];
      ls[warp * 16 + row] = l_part[r];
    }
#pragma unroll
    for (int j = 0; j < NT; ++j)
      if (EXACT || j * 8 < dv) *reinterpret_cast<float2*>(as + ((size_t)warp * 16 + row) * dv + j * 8 + t2) = make_float2(acc[j][2 * r], acc[j][2 * r + 1]);
  }
  __syncthreads();
  for (int i = tid; i < nq * gs * (dv / 2); i += PA_THREADS) {
    const int row = i / (dv / 2), col = (i % (dv / 2)) * 2;
    const float m = fmaxf(fmaxf(ms[row], ms[16 + row]), fmaxf(ms[32 + row], ms[48 + row]));
    float l = 0.f, o0 = 0.f, o1 = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float f = pa_exp2(ms[w * 16 + row] - m);   // zero for a warp that saw nothing (m is finite: every query sees itself)
      const float2 a2 = *reinterpret_cast<const float2*>(as + ((size_t)w * 16 + row) * dv + col);
      l = fmaf(f, ls[w * 16 + row], l);
      o0 = fmaf(f, a2.x, o0);
      o1 = fmaf(f, a2.y, o1);
    }
    const float f = out_factor(g, row0 + row / gs, h_base + row % gs) / l;
    *reinterpret_cast<__nv_bfloat162*>(out + out_row(g, row0 + row / gs) + (size_t)(h_base + row % gs) * dv + col) = __floats2bfloat162_rn(o0 * f, o1 * f);
  }
}

template <int KS, int NT, bool SPLIT>
cudaError_t launch_mma(const void* q, const void* k_cache, const void* v_cache, const void* pk, const void* pv, const AttnSeq* seqs,
                       const LatentTile* tiles, int n_tiles, const int32_t* block_table, int bt_stride, void* out, const PoolAttnGeom& g,
                       cudaStream_t stream) {
  using bf = __nv_bfloat16;
  using SH = PaShape<SPLIT>;
  // the ring; the queries staged before it and the states merged after it are smaller
  const size_t smem = (size_t)SH::NST * SH::CPS * KV_BLOCK * (g.dim + 8 + g.vdim + 8) * sizeof(bf);   // <= 205 KB
  static bool attr_set = false;
  if (!attr_set) {
    const cudaError_t e = cudaFuncSetAttribute(poolattn_mma_kernel<KS, NT, SPLIT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 208 * 1024);
    if (e != cudaSuccess) return e;
    attr_set = true;
  }
  static int group_on = -1;
  if (group_on < 0) {
    const char* e = getenv("TGIS_POOLATTN_GROUP");
    group_on = (e && e[0] == '0') ? 0 : 1;
  }
  const int per_kv = g.heads / g.kv_heads;
  const int gs = (group_on && per_kv <= 16 && 16 % per_kv == 0) ? per_kv : 1;
  const dim3 grid(n_tiles, g.heads / gs, std::max(1, PA_QT * gs / SH::ROWS));
  return launch_k(poolattn_mma_kernel<KS, NT, SPLIT>, grid, dim3(PA_THREADS), smem, stream, reinterpret_cast<const bf*>(q),
                  reinterpret_cast<const bf*>(k_cache), reinterpret_cast<const bf*>(v_cache), reinterpret_cast<const bf*>(pk),
                  reinterpret_cast<const bf*>(pv), seqs, tiles, block_table, bt_stride, reinterpret_cast<bf*>(out), g, gs);
}

bool mma_eligible(const PoolAttnGeom& g, const void* q, const void* k, const void* v, const void* pk, const void* pv, const void* out) {
  static int on = -1;
  if (on < 0) {
    const char* e = getenv("TGIS_POOLATTN_MMA");
    on = (e && e[0] == '0') ? 0 : 1;
  }
  auto al16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  return on && g.dim % 16 == 0 && g.dim <= 16 * MMA_KS && g.vdim % 8 == 0 && g.vdim <= 8 * MMA_MAX_NT && al16(q) && al16(k) && al16(v) &&
         al16(pk) && al16(pv) && al16(out) && g.out_ld % 2 == 0;
}

template <class CT>
cudaError_t launch_fma(const void* q, const void* k_cache, const void* v_cache, const void* pk, const void* pv,
                       const AttnSeq* seqs, const LatentTile* tiles, int n_tiles, const int32_t* block_table, int bt_stride,
                       void* out, const PoolAttnGeom& g, cudaStream_t stream) {
  const size_t smem = ((size_t)PA_QT * g.dim + (size_t)KV_BLOCK * (g.dim + 1) + (size_t)KV_BLOCK * g.vdim + PA_QT * KV_BLOCK +
                       2 * PA_QT) * sizeof(float);
  if (smem > 200 * 1024) return cudaErrorInvalidValue;
  static size_t attr_bytes = 0;   // per instantiation
  if (smem > 48 * 1024 && smem > attr_bytes) {
    const cudaError_t e = cudaFuncSetAttribute(poolattn_kernel<CT, CT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
    attr_bytes = smem;
  }
  return launch_k(poolattn_kernel<CT, CT>, dim3(n_tiles, g.heads), dim3(PA_THREADS), smem, stream,
                  reinterpret_cast<const CT*>(q), reinterpret_cast<const CT*>(k_cache), reinterpret_cast<const CT*>(v_cache),
                  reinterpret_cast<const CT*>(pk), reinterpret_cast<const CT*>(pv), seqs, tiles, block_table, bt_stride,
                  reinterpret_cast<CT*>(out), g);
}

bool geom_ok(const PoolAttnGeom& g) {
  return g.heads >= 1 && g.kv_heads >= 1 && g.heads % g.kv_heads == 0 && g.heads <= 65535 && g.dim >= 1 && g.vdim >= 1 &&
         g.dim <= PREP_MAX_DIM && g.vdim <= POOLATTN_MAX_VDIM && g.rot_dims >= 0 && g.rot_dims <= g.dim && (g.rot_dims & 1) == 0 &&
         (g.pool <= 0 || (g.keep_first <= 0 && g.chunk <= 0));
}

}  // namespace

cudaError_t poolattn_prep_launch(const float* y, int ldy, int q_off, int k_off, int v_off, const float* bias,
                                 const PoolAttnGeom& g, const float* cos_sin, float eps, const int32_t* positions,
                                 const int32_t* slot_mapping, void* q_out, void* k_cache, void* v_cache, int dtype, int T,
                                 cudaStream_t stream) {
  if (T <= 0) return cudaSuccess;
  if (!geom_ok(g) || (g.rot_dims > 0 && cos_sin == nullptr)) return cudaErrorInvalidValue;
  if (v_off == k_off && g.dim != g.vdim) return cudaErrorInvalidValue;
  const dim3 grid(T, (g.heads + 2 * g.kv_heads + PREP_WARPS - 1) / PREP_WARPS);
  using bf = __nv_bfloat16;
  if (g.q_norm != nullptr || g.k_norm != nullptr) {
    if (g.q_norm == nullptr || g.k_norm == nullptr || g.unit_norm) return cudaErrorInvalidValue;
    auto al16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    if (v_off == k_off && (g.rot_interleaved || g.rot_dims == 0) && g.dim % 4 == 0 && g.rot_dims % 4 == 0 && ldy % 4 == 0 && q_off % 4 == 0 &&
        k_off % 4 == 0 && (g.heads + g.kv_heads) * g.dim <= 4 * PREPF_THREADS * PREPF_V && al16(y) && al16(bias) && al16(g.q_norm) &&
        al16(g.k_norm) && al16(cos_sin) && al16(q_out) && al16(k_cache) && al16(v_cache)) {
      if (dtype == DT_BF16)
        return launch_k(poolattn_prep_full_vec_kernel<bf>, dim3(T), dim3(PREPF_THREADS), 0, stream, y, ldy, q_off, k_off, bias, g, cos_sin, eps,
                        positions, slot_mapping, reinterpret_cast<bf*>(q_out), reinterpret_cast<bf*>(k_cache), reinterpret_cast<bf*>(v_cache));
      return launch_k(poolattn_prep_full_vec_kernel<float>, dim3(T), dim3(PREPF_THREADS), 0, stream, y, ldy, q_off, k_off, bias, g, cos_sin, eps,
                      positions, slot_mapping, reinterpret_cast<float*>(q_out), reinterpret_cast<float*>(k_cache), reinterpret_cast<float*>(v_cache));
    }
    const size_t smem = (size_t)(g.heads + g.kv_heads) * g.dim * sizeof(float);
    if (smem > 160 * 1024) return cudaErrorInvalidValue;
    static bool attr_set = false;
    if (smem > 40 * 1024 && !attr_set) {
      cudaError_t e = cudaFuncSetAttribute(poolattn_prep_full_kernel<bf>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
      if (e == cudaSuccess) e = cudaFuncSetAttribute(poolattn_prep_full_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
      if (e != cudaSuccess) return e;
      attr_set = true;
    }
    if (dtype == DT_BF16)
      return launch_k(poolattn_prep_full_kernel<bf>, dim3(T), dim3(PREPF_THREADS), smem, stream, y, ldy, q_off, k_off, v_off, bias, g, cos_sin,
                      eps, positions, slot_mapping, reinterpret_cast<bf*>(q_out), reinterpret_cast<bf*>(k_cache), reinterpret_cast<bf*>(v_cache));
    return launch_k(poolattn_prep_full_kernel<float>, dim3(T), dim3(PREPF_THREADS), smem, stream, y, ldy, q_off, k_off, v_off, bias, g, cos_sin,
                    eps, positions, slot_mapping, reinterpret_cast<float*>(q_out), reinterpret_cast<float*>(k_cache), reinterpret_cast<float*>(v_cache));
  }
  const bool small = g.dim <= 128;   // four entries per lane
  if (dtype == DT_BF16)
    return launch_k(small ? poolattn_prep_kernel<bf, 4> : poolattn_prep_kernel<bf, PREP_MAX_DIM / 32>, grid, dim3(PREP_WARPS * 32), 0,
                    stream, y, ldy, q_off, k_off, v_off, bias, g, cos_sin, eps, positions, slot_mapping, reinterpret_cast<bf*>(q_out),
                    reinterpret_cast<bf*>(k_cache), reinterpret_cast<bf*>(v_cache));
  return launch_k(small ? poolattn_prep_kernel<float, 4> : poolattn_prep_kernel<float, PREP_MAX_DIM / 32>, grid, dim3(PREP_WARPS * 32),
                  0, stream, y, ldy, q_off, k_off, v_off, bias, g, cos_sin, eps, positions, slot_mapping,
                  reinterpret_cast<float*>(q_out), reinterpret_cast<float*>(k_cache), reinterpret_cast<float*>(v_cache));
}

cudaError_t poolattn_pool_launch(const void* k_cache, const void* v_cache, void* pk, void* pv, int dtype,
                                 const AttnSeq* seqs, int n_seqs, const int32_t* block_table, int bt_stride,
                                 const PoolAttnGeom& g, int max_q_len, cudaStream_t stream) {
  if (n_seqs <= 0 || g.pool <= 0 || g.window <= 0) return cudaSuccess;
  if (!geom_ok(g)) return cudaErrorInvalidValue;
  const dim3 grid(n_seqs, std::min(max_q_len / g.pool + 1, 4096));
  if (dtype == DT_BF16)
    return launch_k(poolattn_pool_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream,
                    reinterpret_cast<const __nv_bfloat16*>(k_cache), reinterpret_cast<const __nv_bfloat16*>(v_cache),
                    reinterpret_cast<__nv_bfloat16*>(pk), reinterpret_cast<__nv_bfloat16*>(pv), seqs, block_table, bt_stride, g);
  return launch_k(poolattn_pool_kernel<float>, grid, dim3(128), 0, stream, reinterpret_cast<const float*>(k_cache),
                  reinterpret_cast<const float*>(v_cache), reinterpret_cast<float*>(pk), reinterpret_cast<float*>(pv), seqs,
                  block_table, bt_stride, g);
}

cudaError_t poolattn_launch(const void* q, const void* k_cache, const void* v_cache, const void* pk, const void* pv, int dtype,
                            const AttnSeq* seqs, const LatentTile* tiles, int n_tiles, int n_tokens, const int32_t* block_table,
                            int bt_stride, void* out, int out_dtype, const PoolAttnGeom& g, cudaStream_t stream) {
  if (n_tiles <= 0) return cudaSuccess;
  if (!geom_ok(g) || out_dtype != dtype) return cudaErrorInvalidValue;
  if (dtype == DT_BF16 && mma_eligible(g, q, k_cache, v_cache, pk, pv, out)) {
    const bool split = n_tokens < 4 * n_tiles;   // mostly single tokens
    auto run = [&](auto ks, auto nt) {
      constexpr int KS = decltype(ks)::value, NT = decltype(nt)::value;
      return split ? launch_mma<KS, NT, true>(q, k_cache, v_cache, pk, pv, seqs, tiles, n_tiles, block_table, bt_stride, out, g, stream)
                   : launch_mma<KS, NT, false>(q, k_cache, v_cache, pk, pv, seqs, tiles, n_tiles, block_table, bt_stride, out, g, stream);
    };
    using std::integral_constant;
    if (g.dim == 128 && g.vdim == 128) return run(integral_constant<int, 8>{}, integral_constant<int, 16>{});
    if (g.dim == 64 && g.vdim == 64) return run(integral_constant<int, 4>{}, integral_constant<int, 8>{});
    return g.vdim <= 128 ? run(integral_constant<int, 0>{}, integral_constant<int, 16>{})
                         : run(integral_constant<int, 0>{}, integral_constant<int, MMA_MAX_NT>{});
  }
  if (dtype == DT_BF16)
    return launch_fma<__nv_bfloat16>(q, k_cache, v_cache, pk, pv, seqs, tiles, n_tiles, block_table, bt_stride, out, g, stream);
  return launch_fma<float>(q, k_cache, v_cache, pk, pv, seqs, tiles, n_tiles, block_table, bt_stride, out, g, stream);
}

}  // namespace tgis
