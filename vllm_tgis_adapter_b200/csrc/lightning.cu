// Lightning attention over the portions of a step, chunk by chunk on the tensor cores (kernels.h: LightningChunk).
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

}  // namespace tgis
