// Outer-product memories over the portions of a step, chunk by chunk on the tensor cores: lightning attention and retention (kernels.h:
// LightningChunk) here, gated linear attention (GlaChunk) further down.
// Per head  S_t = r S_{t-1} + k_t v_t^T,  o_t = S_t^T q_t  with one fixed decay r and q, k, v = silu of their projections
// (lightning attention), or q and k rotated by their position and v as projected (retention).  For the n <= 64
// tokens i, j = 0 .. n-1 of a chunk and the state S that the tokens before it left, this is
//     o_i = r^(i+1) S^T q_i + sum_{j <= i} r^(i-j) (q_i . k_j) v_j          S <- r^n S + sum_j r^(n-1-j) k_j v_j^T
// so a portion of T tokens takes T / 64 dependent steps of matrix products instead of T dependent rank-one updates.
//
// One CTA per (sequence, head, 64 value columns), four warps of 16 value columns each.  A warp keeps the TRANSPOSED state [16 values,
// dim] as fp32 accumulator fragments for the whole portion: they are at once the accumulator of the state update (V'^T K) and, lane
// by lane, the B fragments of the read-out (Q S), so the state never passes through shared memory.  The decayed scores are computed
// once per CTA (16 rows per warp) and shared.
//
// silu_cast_kernel (or rotary_rows_kernel) makes q, k and v from the projections once for all CTAs; the chunk after the current one lands in the other half of
// a double buffer.
//
// Precision: q, k and v are rounded to bf16 after silu, as any product input.  Everything the recurrence adds is kept to 32 bits'
// worth: accumulators, state, powers of the decay and the decayed scores are fp32, and where such a number is an operand of a
// product -- the state in the read-out, the decayed scores, the decayed values of the update -- it goes in as the sum of two bf16
// numbers (the rounded one and the rounded rest), two products on the same accumulator.
//
// The chunk grid starts at the portion's first token, so how a prompt was cut changes rounding only.  Slots as in recurrent.cu: the
// state of position 0 is zero, the CTA that reads a piece of a slot's state is the one that rewrites it.
#include <algorithm>
#include <cstdint>
#include <cstdlib>

#include "kernels.h"
#include "launch.cuh"
#include "ptx.cuh"

namespace tgis {
namespace {

using bf = __nv_bfloat16;
constexpr int LC = 64, LV = 64, L_THREADS = 128;   // tokens per chunk, value columns per CTA
constexpr int LDV_ = LV + 8, LDA_ = LC + 8;

__device__ __forceinline__ void l_ldsm_x4(uint32_t (&r)[4], const void* smem) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(smem);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void l_ldsm_x4_trans(uint32_t (&r)[4], const void* smem) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(smem);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void l_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void l_cp_async16(void* smem, const void* gmem) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(a), "l"(gmem) : "memory");
}
// (x, y) as packed bf16 pairs: hi = rounded, lo = the rounded rest
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}

// out[t, i] = silu(x[t, i]), four columns per thread
__global__ void __launch_bounds__(256)
silu_cast_kernel(const float* __restrict__ x, int ldx, bf* __restrict__ out, int ldo, int n) {
  griddep_launch();
  griddep_wait();
  const int t = blockIdx.x;
#pragma unroll 4
  for (int i = (blockIdx.y * 256 + threadIdx.x) * 4; i < n; i += gridDim.y * 1024) {
    const float4 v = *reinterpret_cast<const float4*>(x + (size_t)t * ldx + i);
    // (fast forms: their error is far below the rounding to bf16)
    auto silu = [](float z) { return __fdividef(z, 1.f + __expf(-z)); };
    const __nv_bfloat162 lo = __floats2bfloat162_rn(silu(v.x), silu(v.y)), hi = __floats2bfloat162_rn(silu(v.z), silu(v.w));
    uint2 pk;
    pk.x = *reinterpret_cast<const uint32_t*>(&lo);
    pk.y = *reinterpret_cast<const uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(out + (size_t)t * ldo + i) = pk;
  }
}

// rotary_rows_kernel for heads whose sizes are multiples of eight and rows on 16-byte boundaries: four pairs (or eight entries that pass)
// per thread and step
__global__ void __launch_bounds__(256)
rotary_rows_vec_kernel(RotaryRows a) {
  griddep_launch();
  griddep_wait();
  const int t = blockIdx.x, D = a.dim, half = a.rot_dims / 2, hd = a.heads * D, per = D / 8;
  float* row = a.x + (size_t)t * a.ld;
  const float* cs = a.cos_sin != nullptr ? a.cos_sin + (size_t)a.positions[t] * a.rot_dims : nullptr;
  bf* dst = (a.cast != nullptr && t >= a.n_inplace) ? reinterpret_cast<bf*>(a.cast) + (size_t)t * a.cast_ld : nullptr;
  const int n_v = dst != nullptr ? a.heads * a.vdim / 8 : 0;
  auto put = [&](float* f, bf* b, float4 v) {
    if (b == nullptr) {
      *reinterpret_cast<float4*>(f) = v;
    } else {
      const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
      uint2 pk;
      pk.x = *reinterpret_cast<const uint32_t*>(&lo);
      pk.y = *reinterpret_cast<const uint32_t*>(&hi);
      *reinterpret_cast<uint2*>(b) = pk;
    }
  };
  for (int i = blockIdx.y * 256 + threadIdx.x; i < 2 * a.heads * per + n_v; i += gridDim.y * 256) {
    if (i >= 2 * a.heads * per) {   // values
      const int c = (i - 2 * a.heads * per) * 8;
      put(nullptr, dst + 2 * hd + c, *reinterpret_cast<const float4*>(row + a.v_off + c));
      put(nullptr, dst + 2 * hd + c + 4, *reinterpret_cast<const float4*>(row + a.v_off + c + 4));
      continue;
    }
    const bool is_k = i >= a.heads * per;
    const int r = is_k ? i - a.heads * per : i, h = r / per, e = r % per;
    const float m = is_k ? a.k_mul : a.q_mul;
    const bool turn = e * 4 < half;
    const int p0 = turn ? e * 4 : a.rot_dims + (e * 4 - half) * 2, p1 = turn ? p0 + half : p0 + 4;
    float* src = row + (is_k ? a.k_off : a.q_off) + h * D;
    bf* out = dst != nullptr ? dst + (is_k ? hd : 0) + h * D : nullptr;
    float4 u = *reinterpret_cast<const float4*>(src + p0), v = *reinterpret_cast<const float4*>(src + p1);
    if (turn) {
      const float4 c = *reinterpret_cast<const float4*>(cs + p0), s = *reinterpret_cast<const float4*>(cs + half + p0);
      const float4 u2 = make_float4(u.x * c.x - v.x * s.x, u.y * c.y - v.y * s.y, u.z * c.z - v.z * s.z, u.w * c.w - v.w * s.w);
      v = make_float4(v.x * c.x + u.x * s.x, v.y * c.y + u.y * s.y, v.z * c.z + u.z * s.z, v.w * c.w + u.w * s.w);
      u = u2;
    }
    put(src + p0, out != nullptr ? out + p0 : nullptr, make_float4(u.x * m, u.y * m, u.z * m, u.w * m));
    put(src + p1, out != nullptr ? out + p1 : nullptr, make_float4(v.x * m, v.y * m, v.z * m, v.w * m));
  }
}

// grid (T, y): one token per x; pairs / values of the row in strides of the CTA (kernels.h: RotaryRows)
__global__ void __launch_bounds__(256)
rotary_rows_kernel(RotaryRows a) {
  griddep_launch();
  griddep_wait();
  const int t = blockIdx.x, D = a.dim, half = a.rot_dims / 2, hd = a.heads * D;
  float* row = a.x + (size_t)t * a.ld;
  const float* cs = a.cos_sin != nullptr ? a.cos_sin + (size_t)a.positions[t] * a.rot_dims : nullptr;
  bf* dst = (a.cast != nullptr && t >= a.n_inplace) ? reinterpret_cast<bf*>(a.cast) + (size_t)t * a.cast_ld : nullptr;
  const int per = half + D - a.rot_dims;   // per head: the pairs, then the entries that pass
  const int n_qk = 2 * a.heads * per;
  for (int i = blockIdx.y * 256 + threadIdx.x; i < n_qk; i += gridDim.y * 256) {
    const bool is_k = i >= a.heads * per;
    const int r = is_k ? i - a.heads * per : i, h = r / per, e = r % per;
    const float mul = is_k ? a.k_mul : a.q_mul;
    float* src = row + (is_k ? a.k_off : a.q_off) + h * D;
    bf* out = dst != nullptr ? dst + (is_k ? hd : 0) + h * D : nullptr;
    if (e < half) {
      const float c = cs[e], s = cs[half + e], u = src[e], v = src[e + half];
      const float u2 = (u * c - v * s) * mul, v2 = (v * c + u * s) * mul;
      if (out != nullptr) { out[e] = __float2bfloat16_rn(u2); out[e + half] = __float2bfloat16_rn(v2); }
      else { src[e] = u2; src[e + half] = v2; }
    } else {
      const int p = e - half + a.rot_dims;
      if (out != nullptr) out[p] = __float2bfloat16_rn(src[p] * mul);
      else src[p] *= mul;
    }
  }
  if (dst != nullptr)
    for (int i = blockIdx.y * 256 + threadIdx.x; i < a.heads * a.vdim; i += gridDim.y * 256) dst[2 * hd + i] = __float2bfloat16_rn(row[a.v_off + i]);
}

// DKS: k-steps of 16 over dim (dim <= 16 DKS, a multiple of 16)
template <int DKS>
__global__ void __launch_bounds__(L_THREADS)
lightning_chunk_kernel(LightningChunk a, const AttnSeq* __restrict__ seqs, const int32_t* __restrict__ tok_slot) {
  extern __shared__ __align__(16) uint8_t l_smem[];
  const int D = a.dim, LDQ = D + 8, nks = D / 16;
  const int ring = LC * (2 * LDQ + LDV_);                         // one buffer: Q [LC][LDQ] | K [LC][LDQ] | V [LC][LDV_]
  bf* QKV = reinterpret_cast<bf*>(l_smem);                        // two of them
  bf* Vh = QKV + 2 * ring;                                        // [LC][LDV_]   decayed values, hi and lo
  bf* Vl = Vh + LC * LDV_;
  bf* Ah = Vl + LC * LDV_;                                        // [LC][LDA_]   decayed scores, hi and lo
  bf* Al = Ah + LC * LDA_;
  __shared__ float pw[LC + 1];                                    // r^n
  griddep_launch();
  griddep_wait();
  const AttnSeq sq = seqs[blockIdx.x];
  const int h = blockIdx.y, c0 = blockIdx.z * LV;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, t2 = (lane & 3) * 2;
  const int slot = tok_slot[sq.q_start];
  const bool fresh = sq.kv_len - sq.q_len == 0;
  if (tid <= LC) {
    double p = 1.0, b = (double)a.decay[h];
    for (int n = tid; n > 0; n >>= 1, b *= b)
      if (n & 1) p *= b;
    pw[tid] = (float)p;
  }
  const int n_col = min(LV, a.vdim - c0);   // a multiple of 8
  // the chunk at t0 -> buffer `buf`, 16 bytes per copy; rows up to the next multiple of 16 and columns past the slice are zeros
  const bf* src = reinterpret_cast<const bf*>(a.qkv) + (size_t)h * D;
  const bf* src_v = reinterpret_cast<const bf*>(a.qkv) + a.v_off + (size_t)h * a.vdim + c0;
  auto fetch = [&](int t0, int buf) {
    const int nt = min(LC, sq.q_len - t0), qv = D / 8, per = 2 * qv + LV / 8;
    bf* Qd = QKV + buf * ring;
    for (int t = warp; t < (nt + 15) / 16 * 16; t += L_THREADS / 32) {
      const size_t row = (size_t)(sq.q_start + t0 + t) * a.ld;
      for (int e = lane; e < per; e += 32) {
        const bool is_v = e >= 2 * qv;
        const int c = (is_v ? e - 2 * qv : e < qv ? e : e - qv) * 8;
        bf* dst = is_v ? Qd + LC * 2 * LDQ + t * LDV_ + c : Qd + (e < qv ? 0 : LC * LDQ) + t * LDQ + c;
        if (t < nt && (!is_v || c < n_col)) l_cp_async16(dst, is_v ? src_v + row + c : src + row + (e < qv ? a.q_off : a.k_off) + c);
        else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
      }
    }
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
  fetch(0, 0);
  // S^T fragments: tile n holds rows (value columns) v0 + gq, v0 + gq + 8 and entries 8 n + t2, + 1 of dim
  float S[2 * DKS][4];
  const int v0 = warp * 16;
  float* Sg = a.S + ((size_t)slot * a.heads + h) * D * a.vdim + c0;
#pragma unroll
  for (int n = 0; n < 2 * DKS; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int v = v0 + gq + (e >> 1) * 8, i = n * 8 + t2 + (e & 1);
      S[n][e] = (!fresh && v < n_col && i < D) ? Sg[(size_t)i * a.vdim + v] : 0.f;
    }
  int buf = 0;
  for (int t0 = 0; t0 < sq.q_len; t0 += LC, buf ^= 1) {
    const int nt = min(LC, sq.q_len - t0), n_mt = (nt + 15) / 16;   // rows past nt inside the last 16 are zeros
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    __syncthreads();   // the chunk has landed; the previous chunk's operands are consumed
    if (t0 + LC < sq.q_len) fetch(t0 + LC, buf ^ 1);   // lands while this chunk is worked through
    const bf *Qs = QKV + buf * ring, *Ks = Qs + LC * LDQ, *Vs = Ks + LC * LDQ;
    // ---- decayed values r^(n-1-j) v_j
    for (int t = warp; t < n_mt * 16; t += L_THREADS / 32) {
      static_assert(LV == 64, "one value pair per lane");
      const float2 vf = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(Vs + t * LDV_ + 2 * lane));
      const float p = t < nt ? pw[nt - 1 - t] : 0.f;
      uint32_t hi, lo;
      split2(vf.x * p, vf.y * p, hi, lo);
      *reinterpret_cast<uint32_t*>(Vh + t * LDV_ + 2 * lane) = hi;
      *reinterpret_cast<uint32_t*>(Vl + t * LDV_ + 2 * lane) = lo;
    }
    // ---- decayed scores of this warp's 16 rows
    if (warp < n_mt) {
      float sc[2 * LC / 16][4];
#pragma unroll
      for (int n = 0; n < 2 * LC / 16; ++n) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < DKS; ++ks)
        if (ks < nks) {
          uint32_t qf[4];
          l_ldsm_x4(qf, Qs + (size_t)(warp * 16 + (lane & 15)) * LDQ + ks * 16 + (lane >> 4) * 8);
#pragma unroll
          for (int jj = 0; jj < LC / 16; ++jj)
            if (jj <= warp) {
              uint32_t kf[4];
              l_ldsm_x4(kf, Ks + (size_t)(jj * 16 + (lane >> 4) * 8 + (lane & 7)) * LDQ + ks * 16 + ((lane >> 3) & 1) * 8);
              l_mma(sc[2 * jj], qf, kf[0], kf[1]);
              l_mma(sc[2 * jj + 1], qf, kf[2], kf[3]);
            }
        }
#pragma unroll
      for (int n = 0; n < 2 * LC / 16; ++n)
        if (n / 2 <= warp) {
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            const int i = warp * 16 + gq + r * 8, j = n * 8 + t2;
            const float x = j <= i ? sc[n][2 * r] * pw[i - j] : 0.f, y = j + 1 <= i ? sc[n][2 * r + 1] * pw[i - j - 1] : 0.f;
            uint32_t hi, lo;
            split2(x, y, hi, lo);
            *reinterpret_cast<uint32_t*>(Ah + i * LDA_ + j) = hi;
            *reinterpret_cast<uint32_t*>(Al + i * LDA_ + j) = lo;
          }
        }
    }
    __syncthreads();
    // ---- read-out of the warp's 16 value columns: r^(i+1) Q S, then the chunk's own tokens
    float o[LC / 16][2][4];
#pragma unroll
    for (int mt = 0; mt < LC / 16; ++mt)
#pragma unroll
      for (int n = 0; n < 2; ++n) o[mt][n][0] = o[mt][n][1] = o[mt][n][2] = o[mt][n][3] = 0.f;
    if (!fresh || t0 > 0) {
#pragma unroll
      for (int ks = 0; ks < DKS; ++ks)
        if (ks < nks) {
          uint32_t bh[2][2], bl[2][2];   // [value half][dim half of the k-step]
#pragma unroll
          for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int k = 0; k < 2; ++k) split2(S[2 * ks + k][2 * n], S[2 * ks + k][2 * n + 1], bh[n][k], bl[n][k]);
#pragma unroll
          for (int mt = 0; mt < LC / 16; ++mt)
            if (mt < n_mt) {
              uint32_t qf[4];
              l_ldsm_x4(qf, Qs + (size_t)(mt * 16 + (lane & 15)) * LDQ + ks * 16 + (lane >> 4) * 8);
#pragma unroll
              for (int n = 0; n < 2; ++n) {
                l_mma(o[mt][n], qf, bh[n][0], bh[n][1]);
                l_mma(o[mt][n], qf, bl[n][0], bl[n][1]);
              }
            }
        }
    }
#pragma unroll
    for (int mt = 0; mt < LC / 16; ++mt)
      if (mt < n_mt) {
        const float p0 = pw[mt * 16 + gq + 1], p1 = pw[mt * 16 + gq + 9];
#pragma unroll
        for (int n = 0; n < 2; ++n) { o[mt][n][0] *= p0; o[mt][n][1] *= p0; o[mt][n][2] *= p1; o[mt][n][3] *= p1; }
      }
#pragma unroll
    for (int kk = 0; kk < LC / 16; ++kk)
      if (kk < n_mt) {
        uint32_t vf[4];
        l_ldsm_x4_trans(vf, Vs + (size_t)(kk * 16 + (lane & 15)) * LDV_ + v0 + (lane >> 4) * 8);
#pragma unroll
        for (int mt = kk; mt < LC / 16; ++mt)
          if (mt < n_mt) {
            uint32_t ah[4], al[4];
            l_ldsm_x4(ah, Ah + (size_t)(mt * 16 + (lane & 15)) * LDA_ + kk * 16 + (lane >> 4) * 8);
            l_ldsm_x4(al, Al + (size_t)(mt * 16 + (lane & 15)) * LDA_ + kk * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int n = 0; n < 2; ++n) {
              l_mma(o[mt][n], ah, vf[2 * n], vf[2 * n + 1]);
              l_mma(o[mt][n], al, vf[2 * n], vf[2 * n + 1]);
            }
          }
      }
#pragma unroll
    for (int mt = 0; mt < LC / 16; ++mt)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int t = mt * 16 + gq + r * 8;
        if (t >= nt) continue;
        float* dst = a.out + (size_t)(sq.q_start + t0 + t) * a.ldo + (size_t)h * a.vdim + c0 + v0 + t2;
#pragma unroll
        for (int n = 0; n < 2; ++n)
          if (v0 + n * 8 < n_col) *reinterpret_cast<float2*>(dst + n * 8) = make_float2(o[mt][n][2 * r], o[mt][n][2 * r + 1]);
      }
    // ---- the state behind the chunk: r^n S + V'^T K
    const float pn = pw[nt];
#pragma unroll
    for (int n = 0; n < 2 * DKS; ++n) { S[n][0] *= pn; S[n][1] *= pn; S[n][2] *= pn; S[n][3] *= pn; }
#pragma unroll
    for (int kk = 0; kk < LC / 16; ++kk)
      if (kk < n_mt) {
        uint32_t vh[4], vl[4];   // A fragments of V'^T: rows = values, k = tokens
        const size_t at = (size_t)(kk * 16 + (lane & 7) + (lane >> 4) * 8) * LDV_ + v0 + ((lane >> 3) & 1) * 8;
        l_ldsm_x4_trans(vh, Vh + at);
        l_ldsm_x4_trans(vl, Vl + at);
#pragma unroll
        for (int ks = 0; ks < DKS; ++ks)
          if (ks < nks) {
            uint32_t kf[4];
            l_ldsm_x4_trans(kf, Ks + (size_t)(kk * 16 + (lane & 15)) * LDQ + ks * 16 + (lane >> 4) * 8);
            l_mma(S[2 * ks], vh, kf[0], kf[1]);
            l_mma(S[2 * ks + 1], vh, kf[2], kf[3]);
            l_mma(S[2 * ks], vl, kf[0], kf[1]);
            l_mma(S[2 * ks + 1], vl, kf[2], kf[3]);
          }
      }
  }
#pragma unroll
  for (int n = 0; n < 2 * DKS; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int v = v0 + gq + (e >> 1) * 8, i = n * 8 + t2 + (e & 1);
      if (v < n_col && i < D) Sg[(size_t)i * a.vdim + v] = S[n][e];
    }
}

template <int DKS>
cudaError_t launch_chunks(const LightningChunk& a, const AttnSeq* seqs, int n_seqs, const int32_t* tok_slot, cudaStream_t stream) {
  const size_t smem = (size_t)LC * (2 * (2 * (a.dim + 8) + LDV_) + 2 * LDV_ + 2 * LDA_) * sizeof(bf);   // <= 122 KB
  static bool attr_set = false;
  if (!attr_set) {
    const cudaError_t e = cudaFuncSetAttribute(lightning_chunk_kernel<DKS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
    if (e != cudaSuccess) return e;
    attr_set = true;
  }
  return launch_k(lightning_chunk_kernel<DKS>, dim3(n_seqs, a.heads, (a.vdim + LV - 1) / LV), dim3(L_THREADS), smem, stream, a, seqs, tok_slot);
}

// ---------------------------------------------------------------------------------------------------------------- gated linear attention
// Per head  S_t = diag(f_t) S_{t-1} + k_t v_t^T,  o_t = S_t^T q_t  with a decay f_t per key channel (kernels.h: GlaChunk).  For the n <= GC
// tokens of a chunk, with F(j, i] the product of f over the tokens j + 1 .. i (per channel) and S what the tokens before left,
//     o_i = (q_i F(-1, i])^T S + sum_{j <= i} A_ij v_j,   A_ij = sum_c q_ic k_jc F(j, i]_c
//     S  <- diag(F(-1, n - 1]) S + sum_j (k_j F(j, n - 1]) v_j^T
// Every factor is a product of decays over an INTERVAL: nothing is ever divided by a decay, so strong decays cannot overflow.  Two
// kernels:
//   gla_prep_kernel   all chunks of the step at once: decays from their low-rank map, prefix and suffix products, the decayed queries
//                     and keys, and the chunk's scores A -- inside 16-token blocks by running products in fp32 (a lane owns channels,
//                     32 scores are reduced over the lanes together), between the two blocks as a product of operands decayed to the
//                     border between them
//   gla_chunk_kernel  the recurrence over a portion's chunks, as lightning_chunk_kernel: a warp owns 16 value columns and keeps the
//                     transposed state in accumulator fragments
// What carries decays goes into products as the sum of two bf16 numbers; v is rounded to bf16 once, q and k are not rounded.
constexpr int GC = GLA_CHUNK, GB = 16, G_THREADS = 128;
static_assert(GC == 2 * GB, "one off-diagonal block per chunk");
constexpr int LDGA = GC + 8;

__device__ __forceinline__ float l_logsigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// lane l leaves with the sum over all lanes of v[l]
__device__ __forceinline__ float reduce32(float (&v)[32], int lane) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const bool up = (lane & o) != 0;
#pragma unroll
    for (int n = 0; n < o; ++n) {
      const float keep = up ? v[n + o] : v[n], send = up ? v[n] : v[n + o];
      v[n] = keep + __shfl_xor_sync(0xffffffffu, send, o);
    }
  }
  return v[0];
}
template <int DPL>
__device__ __forceinline__ void ld_row(float (&r)[DPL], const float* p, bool live) {
  if (DPL == 4) {
    const float4 x = live ? *reinterpret_cast<const float4*>(p) : make_float4(0.f, 0.f, 0.f, 0.f);
    r[0] = x.x; r[1] = x.y; r[2 % DPL] = x.z; r[3 % DPL] = x.w;
  } else {
    const float2 x = live ? *reinterpret_cast<const float2*>(p) : make_float2(0.f, 0.f);
    r[0] = x.x; r[1] = x.y;
  }
}
// scores of rows [I0, I1) of one 16-token block: pair p = i (i + 1) / 2 + delta is A[i][i - delta]; rows of q / k / f are ldf floats apart
template <int I0, int I1, int DPL>
__device__ __forceinline__ void gla_block_scores(const float* q, const float* k, const float* f, int ldf, float* A, int lda, int D, int lane) {
  float kr[I1][DPL], fr[I1][DPL];
  const bool live = lane * DPL < D;
#pragma unroll
  for (int j = 0; j < I1; ++j) {
    ld_row<DPL>(kr[j], k + j * ldf + lane * DPL, live);
    ld_row<DPL>(fr[j], f + j * ldf + lane * DPL, live);
  }
  constexpr int P0 = I0 * (I0 + 1) / 2, P1 = I1 * (I1 + 1) / 2;
  float v[32];
#pragma unroll
  for (int i = I0; i < I1; ++i) {
    float cur[DPL];
    ld_row<DPL>(cur, q + i * ldf + lane * DPL, live);
#pragma unroll
    for (int dl = 0; dl <= i; ++dl) {
      const int p = i * (i + 1) / 2 + dl, n = (p - P0) & 31, j = i - dl;
      float s = 0.f;
#pragma unroll
      for (int e = 0; e < DPL; ++e) {
        s = fmaf(cur[e], kr[j][e], s);
        cur[e] *= fr[j][e];
      }
      v[n] = s;
      if (n == 31 || p == P1 - 1) {
#pragma unroll
        for (int z = 0; z < 32; ++z)
          if (z > n) v[z] = 0.f;
        const float tot = reduce32(v, lane);
        const int mine = p - n + lane;   // the pair whose sum this lane holds
        if (mine < P1) {
          const int r = (int)((sqrtf(8.f * (float)mine + 1.f) - 1.f) * 0.5f);   // (exact: 8 p + 1 is a square where r steps)
          A[r * lda + r - (mine - r * (r + 1) / 2)] = tot;
        }
      }
    }
  }
}

// grid (16-token tiles, heads): the CTA of a tile whose first token opens a chunk of its portion takes the chunk's GC tokens
template <int DPL>
__global__ void __launch_bounds__(G_THREADS, 3)
gla_prep_kernel(GlaChunk a, const AttnSeq* __restrict__ seqs, const LatentTile* __restrict__ tiles, int first_seq) {
  extern __shared__ __align__(16) uint8_t g_smem[];
  griddep_launch();
  griddep_wait();
  const LatentTile tl = tiles[blockIdx.x];
  if (tl.q0 % GC != 0 || tl.seq < first_seq) return;
  const AttnSeq sq = seqs[tl.seq];
  const int nt = min(GC, sq.q_len - tl.q0), row0 = sq.q_start + tl.q0, h = blockIdx.y;
  const int D = a.dim, LD = D + 4, LDQ = D + 8, R = a.rank;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  float* fs = reinterpret_cast<float*>(g_smem);   // [GC][LD] decays (1 past the chunk)
  float* qs = fs + GC * LD;                       // [GC][LD]
  float* ks = qs + GC * LD;                       // [GC][LD]
  float* As = ks + GC * LD;                       // [GC][GC + 1]
  bf* qlh = reinterpret_cast<bf*>(As + GC * (GC + 1) + (GC * (GC + 1)) % 4);   // [GB][LDQ] second block's queries decayed from its start
  bf* qll = qlh + GB * LDQ;
  bf* klh = qll + GB * LDQ;                       // [GB][LDQ] first block's keys decayed to its end
  bf* kll = klh + GB * LDQ;
  float* a1s = reinterpret_cast<float*>(qlh);     // [R][GC], consumed before qlh is written, and
  float* a2s = a1s + R * GC;                      // [R][D + 2]
  // (read-only inputs through __ldg: their loads may pass the stores)
  const int c2 = (tid & 63) * 2, half = tid >> 6;   // two channels; half 0: tokens 0..15 / queries, half 1: tokens 16..31 / keys
  const bool ch_ok = c2 < D;
  {
    float2 xr[GC];
    const float* src = (half == 0 ? a.q : a.k) + (size_t)row0 * a.ld + (size_t)h * D + c2;
#pragma unroll
    for (int t = 0; t < GC; ++t) xr[t] = ch_ok && t < nt ? __ldg(reinterpret_cast<const float2*>(src + (size_t)t * a.ld)) : make_float2(0.f, 0.f);
#pragma unroll 4
    for (int i = tid; i < GC * R; i += G_THREADS) {
      const int t = i / R;
      a1s[(i % R) * GC + t] = t < nt ? __ldg(a.a1 + (size_t)(row0 + t) * a.ld + i % R) : 0.f;
    }
    const uint16_t* w2 = reinterpret_cast<const uint16_t*>(a.a2) + (size_t)h * D * R;
#pragma unroll 8
    for (int i = tid; i < D * R; i += G_THREADS) a2s[(i % R) * (D + 2) + i / R] = __uint_as_float((uint32_t)__ldg(w2 + i) << 16);
    if (ch_ok) {
      float* dst = (half == 0 ? qs : ks) + c2;
      const float m = half == 0 ? a.q_scale : 1.f;
#pragma unroll
      for (int t = 0; t < GC; ++t) *reinterpret_cast<float2*>(dst + t * LD) = make_float2(xr[t].x * m, xr[t].y * m);
    }
  }
  __syncthreads();
  if (ch_ok) {
    const size_t hc = (size_t)h * D + c2;
    float z0[GB], z1[GB];
    const float b0 = a.bias[hc], b1 = a.bias[hc + 1];
#pragma unroll
    for (int t = 0; t < GB; ++t) { z0[t] = b0; z1[t] = b1; }
    for (int r = 0; r < R; ++r) {
      const float2 x = *reinterpret_cast<const float2*>(a2s + r * (D + 2) + c2);
#pragma unroll
      for (int t = 0; t < GB; t += 4) {
        const float4 y = *reinterpret_cast<const float4*>(a1s + r * GC + half * GB + t);
        z0[t] = fmaf(y.x, x.x, z0[t]); z1[t] = fmaf(y.x, x.y, z1[t]);
        z0[t + 1] = fmaf(y.y, x.x, z0[t + 1]); z1[t + 1] = fmaf(y.y, x.y, z1[t + 1]);
        z0[t + 2] = fmaf(y.z, x.x, z0[t + 2]); z1[t + 2] = fmaf(y.z, x.y, z1[t + 2]);
        z0[t + 3] = fmaf(y.w, x.x, z0[t + 3]); z1[t + 3] = fmaf(y.w, x.y, z1[t + 3]);
      }
    }
#pragma unroll
    for (int t = 0; t < GB; ++t) {
      const int tt = half * GB + t;
      float2 f = make_float2(1.f, 1.f);
      if (tt < nt) f = make_float2(expf(l_logsigmoid(z0[t]) * a.inv_tau), expf(l_logsigmoid(z1[t]) * a.inv_tau));
      *reinterpret_cast<float2*>(fs + tt * LD + c2) = f;
    }
  }
  __syncthreads();
  const int W = gla_row(D);
  bf* ops = reinterpret_cast<bf*>(a.ops);
  auto put = [&](bf* hi, bf* lo, float x, float y) {
    uint32_t ph, pl;
    split2(x, y, ph, pl);
    *reinterpret_cast<uint32_t*>(hi) = ph;
    *reinterpret_cast<uint32_t*>(lo) = pl;
  };
  if (ch_ok && half == 0) {   // queries, forward
    float p0 = 1.f, p1 = 1.f, l0 = 1.f, l1 = 1.f;
#pragma unroll 4
    for (int t = 0; t < GC; ++t) {
      const float2 x = *reinterpret_cast<const float2*>(qs + t * LD + c2);
      const float2 f = *reinterpret_cast<const float2*>(fs + t * LD + c2);
      p0 *= f.x;
      p1 *= f.y;
      if (t >= GB) {
        l0 *= f.x;
        l1 *= f.y;
        put(qlh + (t - GB) * LDQ + c2, qll + (t - GB) * LDQ + c2, x.x * l0, x.y * l1);
      }
      if (t < nt) {
        bf* o = ops + ((size_t)(row0 + t) * a.heads + h) * W + c2;
        put(o, o + D, x.x * p0, x.y * p1);
      }
    }
    *reinterpret_cast<float2*>(a.chunk_decay + (size_t)row0 * a.heads * D + (size_t)h * D + c2) = make_float2(p0, p1);
  } else if (ch_ok) {         // keys, backward
    float p0 = 1.f, p1 = 1.f, l0 = 1.f, l1 = 1.f;
#pragma unroll 4
    for (int t = GC - 1; t >= 0; --t) {
      const float2 x = *reinterpret_cast<const float2*>(ks + t * LD + c2);
      const float2 f = *reinterpret_cast<const float2*>(fs + t * LD + c2);
      if (t < nt) {
        bf* o = ops + ((size_t)(row0 + t) * a.heads + h) * W + 2 * D + c2;
        put(o, o + D, x.x * p0, x.y * p1);
      }
      p0 *= f.x;
      p1 *= f.y;
      if (t < GB) {
        put(klh + t * LDQ + c2, kll + t * LDQ + c2, x.x * l0, x.y * l1);
        l0 *= f.x;
        l1 *= f.y;
      }
    }
  }
  const int v4 = a.vdim / 4;
#pragma unroll 4
  for (int i = tid; i < nt * v4; i += G_THREADS) {   // the values, rounded once
    const int t = i / v4, c = i % v4 * 4;
    const float* src = a.v + (size_t)(row0 + t) * a.ld + (size_t)h * a.vdim + c;
    const float2 x = __ldg(reinterpret_cast<const float2*>(src)), y = __ldg(reinterpret_cast<const float2*>(src + 2));
    const __nv_bfloat162 lo = __floats2bfloat162_rn(x.x, x.y), hi = __floats2bfloat162_rn(y.x, y.y);
    uint2 pk;
    pk.x = *reinterpret_cast<const uint32_t*>(&lo);
    pk.y = *reinterpret_cast<const uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(reinterpret_cast<bf*>(a.vb) + (size_t)(row0 + t) * a.heads * a.vdim + (size_t)h * a.vdim + c) = pk;
  }
  __syncthreads();
  // ---- scores: warps 0 and 1 the first block (rows 0..10 | 11..15: as many pairs each), warps 2 and 3 the second
  const int blk = warp >> 1, b0 = blk * GB;
  if (b0 < nt) {
    const float *qb = qs + b0 * LD, *kb = ks + b0 * LD, *fb = fs + b0 * LD;
    float* Ab = As + b0 * (GC + 1) + b0;
    if ((warp & 1) == 0) gla_block_scores<0, 11, DPL>(qb, kb, fb, LD, Ab, GC + 1, D, lane);
    else gla_block_scores<11, 16, DPL>(qb, kb, fb, LD, Ab, GC + 1, D, lane);
  }
  if (warp < 2 && nt > GB) {   // second block's rows x first block's keys 8 warp .. 8 warp + 7
    float s[4] = {0.f, 0.f, 0.f, 0.f};
    for (int k0 = 0; k0 < D; k0 += 16) {
      uint32_t qh[4], ql[4], kh[4], kl[4];
      const size_t qa = (size_t)(lane & 15) * LDQ + k0 + (lane >> 4) * 8, ka = (size_t)((lane >> 4) * 8 + (lane & 7)) * LDQ + k0 + ((lane >> 3) & 1) * 8;
      l_ldsm_x4(qh, qlh + qa);
      l_ldsm_x4(ql, qll + qa);
      l_ldsm_x4(kh, klh + ka);
      l_ldsm_x4(kl, kll + ka);
      l_mma(s, qh, kh[2 * warp], kh[2 * warp + 1]);
      l_mma(s, qh, kl[2 * warp], kl[2 * warp + 1]);
      l_mma(s, ql, kh[2 * warp], kh[2 * warp + 1]);
    }
    const int g = lane >> 2, t2 = (lane & 3) * 2 + 8 * warp;
    As[(GB + g) * (GC + 1) + t2] = s[0];
    As[(GB + g) * (GC + 1) + t2 + 1] = s[1];
    As[(GB + g + 8) * (GC + 1) + t2] = s[2];
    As[(GB + g + 8) * (GC + 1) + t2 + 1] = s[3];
  }
  __syncthreads();
  for (int i = tid; i < nt * (GC / 2); i += G_THREADS) {
    const int t = i / (GC / 2), j = i % (GC / 2) * 2;
    bf* o = ops + ((size_t)(row0 + t) * a.heads + h) * W + 4 * D + j;
    put(o, o + GC, j <= t ? As[t * (GC + 1) + j] : 0.f, j + 1 <= t ? As[t * (GC + 1) + j + 1] : 0.f);
  }
}

// grid (sequences, heads, 64-column slices), four warps of 16 value columns; DKS as above
template <int DKS>
__global__ void __launch_bounds__(L_THREADS)
gla_chunk_kernel(GlaChunk a, const AttnSeq* __restrict__ seqs, const int32_t* __restrict__ tok_slot) {
  extern __shared__ __align__(16) uint8_t l_smem[];
  const int D = a.dim, LDQ = D + 8, nks = D / 16, W = gla_row(D);
  const int ring = GC * (4 * LDQ + LDV_ + 2 * LDGA);   // one buffer: Q hi | Q lo | K hi | K lo [GC][LDQ] each | V [GC][LDV_] | A hi | A lo [GC][LDGA]
  bf* RB = reinterpret_cast<bf*>(l_smem);              // two of them
  float* EB = reinterpret_cast<float*>(RB + 2 * ring); // [2][D] the chunk's whole decay
  griddep_launch();
  griddep_wait();
  const AttnSeq sq = seqs[blockIdx.x];
  const int h = blockIdx.y, c0 = blockIdx.z * LV;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, t2 = (lane & 3) * 2;
  const int slot = tok_slot[sq.q_start];
  const bool fresh = sq.kv_len - sq.q_len == 0;
  const int n_col = min(LV, a.vdim - c0);   // a multiple of 8
  const bf* ops = reinterpret_cast<const bf*>(a.ops) + (size_t)h * W;
  const bf* vb = reinterpret_cast<const bf*>(a.vb) + (size_t)h * a.vdim + c0;
  // a row of a chunk is `per` 16-byte pieces, a lane's are lane, lane + 32, ..: where each comes from and goes to (kind 0: none,
  // 1: decayed queries, keys and scores, 2: values, 3: a value column past the slice -- zeros)
  constexpr int PPL = (2 * DKS * 4 + 2 * GC / 8 + LV / 8 + 31) / 32;
  int p_kind[PPL], p_dst[PPL], p_ld[PPL], p_src[PPL];
#pragma unroll
  for (int i = 0; i < PPL; ++i) {
    const int e = lane + 32 * i, qv = D / 8, av = GC / 8;
    p_kind[i] = p_dst[i] = p_ld[i] = p_src[i] = 0;
    if (e < 4 * qv) {
      p_kind[i] = 1; p_src[i] = e * 8; p_ld[i] = LDQ; p_dst[i] = e / qv * GC * LDQ + e % qv * 8;
    } else if (e < 4 * qv + 2 * av) {
      const int x = e - 4 * qv;
      p_kind[i] = 1; p_src[i] = e * 8; p_ld[i] = LDGA; p_dst[i] = GC * (4 * LDQ + LDV_) + x / av * GC * LDGA + x % av * 8;
    } else if (e < 4 * qv + 2 * av + LV / 8) {
      const int c = (e - 4 * qv - 2 * av) * 8;
      p_kind[i] = c < n_col ? 2 : 3; p_src[i] = c; p_ld[i] = LDV_; p_dst[i] = GC * 4 * LDQ + c;
    }
  }
  auto fetch = [&](int t0, int buf) {   // rows up to the next multiple of 16 and columns past the slice are zeros
    const int nt = min(GC, sq.q_len - t0);
    bf* B = RB + buf * ring;
    const bf* o_row = ops + (size_t)(sq.q_start + t0) * a.heads * W;
    const bf* v_row = vb + (size_t)(sq.q_start + t0) * a.heads * a.vdim;
    for (int t = warp; t < (nt + 15) / 16 * 16; t += L_THREADS / 32) {
#pragma unroll
      for (int i = 0; i < PPL; ++i) {
        if (p_kind[i] == 0) continue;
        bf* dst = B + p_dst[i] + t * p_ld[i];
        if (t < nt && p_kind[i] < 3) l_cp_async16(dst, (p_kind[i] == 1 ? o_row + (size_t)t * a.heads * W : v_row + (size_t)t * a.heads * a.vdim) + p_src[i]);
        else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
      }
    }
    for (int e = tid; e < D / 4; e += L_THREADS) l_cp_async16(EB + buf * D + e * 4, a.chunk_decay + ((size_t)(sq.q_start + t0) * a.heads + h) * D + e * 4);
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
  fetch(0, 0);
  // S^T fragments: tile n holds rows (value columns) v0 + gq, v0 + gq + 8 and entries 8 n + t2, + 1 of dim
  float S[2 * DKS][4];
  const int v0 = warp * 16;
  float* Sg = a.S + ((size_t)slot * a.heads + h) * D * a.vdim + c0;
#pragma unroll
  for (int n = 0; n < 2 * DKS; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int v = v0 + gq + (e >> 1) * 8, i = n * 8 + t2 + (e & 1);
      S[n][e] = (!fresh && v < n_col && i < D) ? Sg[(size_t)i * a.vdim + v] : 0.f;
    }
  int buf = 0;
  for (int t0 = 0; t0 < sq.q_len; t0 += GC, buf ^= 1) {
    const int nt = min(GC, sq.q_len - t0), n_mt = (nt + 15) / 16;   // rows past nt inside the last 16 are zeros
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    __syncthreads();   // the chunk has landed; the previous chunk's operands are consumed
    if (t0 + GC < sq.q_len) fetch(t0 + GC, buf ^ 1);   // lands while this chunk is worked through
    const bf *Qh = RB + buf * ring, *Ql = Qh + GC * LDQ, *Kh = Ql + GC * LDQ, *Kl = Kh + GC * LDQ, *Vs = Kl + GC * LDQ, *Ah = Vs + GC * LDV_,
             *Al = Ah + GC * LDGA;
    const float* E = EB + buf * D;
    // ---- read-out of the warp's 16 value columns: decayed queries times the state, then the chunk's own tokens
    float o[GC / 16][2][4];
#pragma unroll
    for (int mt = 0; mt < GC / 16; ++mt)
#pragma unroll
      for (int n = 0; n < 2; ++n) o[mt][n][0] = o[mt][n][1] = o[mt][n][2] = o[mt][n][3] = 0.f;
    if (!fresh || t0 > 0) {
#pragma unroll
      for (int ks = 0; ks < DKS; ++ks)
        if (ks < nks) {
          uint32_t bh[2][2], bl[2][2];   // [value half][dim half of the k-step]
#pragma unroll
          for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int k = 0; k < 2; ++k) split2(S[2 * ks + k][2 * n], S[2 * ks + k][2 * n + 1], bh[n][k], bl[n][k]);
#pragma unroll
          for (int mt = 0; mt < GC / 16; ++mt)
            if (mt < n_mt) {
              uint32_t qh[4], ql[4];
              const size_t at = (size_t)(mt * 16 + (lane & 15)) * LDQ + ks * 16 + (lane >> 4) * 8;
              l_ldsm_x4(qh, Qh + at);
              l_ldsm_x4(ql, Ql + at);
#pragma unroll
              for (int n = 0; n < 2; ++n) {
                l_mma(o[mt][n], qh, bh[n][0], bh[n][1]);
                l_mma(o[mt][n], qh, bl[n][0], bl[n][1]);
                l_mma(o[mt][n], ql, bh[n][0], bh[n][1]);
              }
            }
        }
    }
#pragma unroll
    for (int kk = 0; kk < GC / 16; ++kk)
      if (kk < n_mt) {
        uint32_t vf[4];
        l_ldsm_x4_trans(vf, Vs + (size_t)(kk * 16 + (lane & 15)) * LDV_ + v0 + (lane >> 4) * 8);
#pragma unroll
        for (int mt = kk; mt < GC / 16; ++mt)
          if (mt < n_mt) {
            uint32_t ah[4], al[4];
            const size_t at = (size_t)(mt * 16 + (lane & 15)) * LDGA + kk * 16 + (lane >> 4) * 8;
            l_ldsm_x4(ah, Ah + at);
            l_ldsm_x4(al, Al + at);
#pragma unroll
            for (int n = 0; n < 2; ++n) {
              l_mma(o[mt][n], ah, vf[2 * n], vf[2 * n + 1]);
              l_mma(o[mt][n], al, vf[2 * n], vf[2 * n + 1]);
            }
          }
      }
#pragma unroll
    for (int mt = 0; mt < GC / 16; ++mt)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int t = mt * 16 + gq + r * 8;
        if (t >= nt) continue;
        float* dst = a.out + (size_t)(sq.q_start + t0 + t) * a.ldo + (size_t)h * a.vdim + c0 + v0 + t2;
#pragma unroll
        for (int n = 0; n < 2; ++n)
          if (v0 + n * 8 < n_col) *reinterpret_cast<float2*>(dst + n * 8) = make_float2(o[mt][n][2 * r], o[mt][n][2 * r + 1]);
      }
    // ---- the state behind the chunk: its whole decay per channel, then V^T K
#pragma unroll
    for (int n = 0; n < 2 * DKS; ++n)
      if (n < 2 * nks) {
        const float2 f = *reinterpret_cast<const float2*>(E + n * 8 + t2);
        S[n][0] *= f.x; S[n][1] *= f.y; S[n][2] *= f.x; S[n][3] *= f.y;
      }
#pragma unroll
    for (int kk = 0; kk < GC / 16; ++kk)
      if (kk < n_mt) {
        uint32_t va[4];   // A fragments of V^T: rows = values, k = tokens
        l_ldsm_x4_trans(va, Vs + (size_t)(kk * 16 + (lane & 7) + (lane >> 4) * 8) * LDV_ + v0 + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int ks = 0; ks < DKS; ++ks)
          if (ks < nks) {
            uint32_t kh[4], kl[4];
            const size_t at = (size_t)(kk * 16 + (lane & 15)) * LDQ + ks * 16 + (lane >> 4) * 8;
            l_ldsm_x4_trans(kh, Kh + at);
            l_ldsm_x4_trans(kl, Kl + at);
            l_mma(S[2 * ks], va, kh[0], kh[1]);
            l_mma(S[2 * ks + 1], va, kh[2], kh[3]);
            l_mma(S[2 * ks], va, kl[0], kl[1]);
            l_mma(S[2 * ks + 1], va, kl[2], kl[3]);
          }
      }
  }
#pragma unroll
  for (int n = 0; n < 2 * DKS; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int v = v0 + gq + (e >> 1) * 8, i = n * 8 + t2 + (e & 1);
      if (v < n_col && i < D) Sg[(size_t)i * a.vdim + v] = S[n][e];
    }
}

template <int DKS>
cudaError_t launch_gla(const GlaChunk& a, const AttnSeq* seqs, int first_seq, int n_seqs, const LatentTile* tiles, int n_tiles,
                       const int32_t* tok_slot, cudaStream_t stream) {
  constexpr int DPL = DKS <= 4 ? 2 : 4;
  const size_t tail = std::max((size_t)4 * GB * (a.dim + 8) * sizeof(bf), (size_t)a.rank * (GC + a.dim + 2) * sizeof(float));
  const size_t smem_p = ((size_t)3 * GC * (a.dim + 4) + GC * (GC + 1)) * sizeof(float) + tail;                       // <= 97 KB (73 KB up to a rank of 26)
  const size_t smem_c = (size_t)2 * GC * (4 * (a.dim + 8) + LDV_ + 2 * LDGA) * sizeof(bf) + (size_t)2 * a.dim * sizeof(float);   // <= 90 KB
  static bool attr_set = false;
  if (!attr_set) {
    cudaError_t e = cudaFuncSetAttribute(gla_prep_kernel<DPL>, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(gla_chunk_kernel<DKS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024);
    if (e != cudaSuccess) return e;
    attr_set = true;
  }
  const cudaError_t e = launch_k(gla_prep_kernel<DPL>, dim3(n_tiles, a.heads), dim3(G_THREADS), smem_p, stream, a, seqs, tiles, first_seq);
  if (e != cudaSuccess) return e;
  return launch_k(gla_chunk_kernel<DKS>, dim3(n_seqs - first_seq, a.heads, (a.vdim + LV - 1) / LV), dim3(L_THREADS), smem_c, stream, a, seqs + first_seq,
                  tok_slot);
}

}  // namespace

bool lightning_chunk_eligible(int dim, int vdim) {
  static int on = -1;
  if (on < 0) {
    const char* e = getenv("TGIS_LIGHTNING_CHUNK");
    on = (e && e[0] == '0') ? 0 : 1;
  }
  return on && dim % 16 == 0 && dim >= 16 && dim <= 128 && vdim % 8 == 0 && vdim >= 8;
}

cudaError_t silu_cast_launch(const float* x, int ldx, void* out, int ldo, int n, int T, cudaStream_t stream) {
  if (T <= 0 || n <= 0) return cudaSuccess;
  if (n % 4 != 0 || ldx % 4 != 0 || ldo % 4 != 0 || (reinterpret_cast<uintptr_t>(x) & 15) != 0 || (reinterpret_cast<uintptr_t>(out) & 7) != 0)
    return cudaErrorInvalidValue;
  return launch_k(silu_cast_kernel, dim3(T, std::min((n + 1023) / 1024, 2)), dim3(256), 0, stream, x, ldx, reinterpret_cast<bf*>(out), ldo, n);
}

cudaError_t rotary_rows_launch(const RotaryRows& a, int T, cudaStream_t stream) {
  if (T <= 0) return cudaSuccess;
  if (a.heads < 1 || a.dim < 1 || a.rot_dims < 0 || a.rot_dims > a.dim || (a.rot_dims & 1) || (a.rot_dims > 0 && a.cos_sin == nullptr))
    return cudaErrorInvalidValue;
  auto al16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  if (a.dim % 8 == 0 && a.rot_dims % 8 == 0 && a.vdim % 8 == 0 && a.ld % 4 == 0 && a.q_off % 4 == 0 && a.k_off % 4 == 0 && a.v_off % 4 == 0 &&
      a.cast_ld % 8 == 0 && al16(a.x) && al16(a.cast) && al16(a.cos_sin))
    return launch_k(rotary_rows_vec_kernel, dim3(T, std::min((a.heads * (2 * a.dim + a.vdim) + 2047) / 2048, 8)), dim3(256), 0, stream, a);
  return launch_k(rotary_rows_kernel, dim3(T, std::min((a.heads * a.dim + 511) / 512, 8)), dim3(256), 0, stream, a);
}

cudaError_t lightning_chunk_launch(const LightningChunk& a, const AttnSeq* seqs, int n_seqs, const int32_t* tok_slot, cudaStream_t stream) {
  if (n_seqs <= 0) return cudaSuccess;
  if (!lightning_chunk_eligible(a.dim, a.vdim) || a.heads < 1 || a.heads > 65535 || a.decay == nullptr || a.ld % 8 != 0 || a.q_off % 8 != 0 ||
      a.k_off % 8 != 0 || a.v_off % 8 != 0 || a.ldo % 2 != 0 || (reinterpret_cast<uintptr_t>(a.qkv) & 15) != 0 ||
      (reinterpret_cast<uintptr_t>(a.out) & 7) != 0)
    return cudaErrorInvalidValue;
  return a.dim <= 64 ? launch_chunks<4>(a, seqs, n_seqs, tok_slot, stream) : launch_chunks<8>(a, seqs, n_seqs, tok_slot, stream);
}

bool gla_chunk_eligible(int dim, int vdim, int rank) { return lightning_chunk_eligible(dim, vdim) && rank >= 1 && rank <= 64; }

cudaError_t gla_chunk_launch(const GlaChunk& a, const AttnSeq* seqs, int first_seq, int n_seqs, const LatentTile* tiles, int n_tiles,
                             const int32_t* tok_slot, cudaStream_t stream) {
  if (n_seqs <= first_seq || n_tiles <= 0) return cudaSuccess;
  auto al = [](const void* p, int n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; };
  if (!gla_chunk_eligible(a.dim, a.vdim, a.rank) || a.heads < 1 || a.heads > 65535 || a.ld % 2 != 0 || !al(a.q, 8) || !al(a.k, 8) || !al(a.v, 8) ||
      !al(a.ops, 16) || !al(a.vb, 16) || !al(a.chunk_decay, 16) || !al(a.out, 8) || a.ldo % 2 != 0 || a.bias == nullptr || !(a.inv_tau > 0.f))
    return cudaErrorInvalidValue;
  return a.dim <= 64 ? launch_gla<4>(a, seqs, first_seq, n_seqs, tiles, n_tiles, tok_slot, stream)
                     : launch_gla<8>(a, seqs, first_seq, n_seqs, tiles, n_tiles, tok_slot, stream);
}

}  // namespace tgis
