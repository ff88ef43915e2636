// Mixture-of-experts bookkeeping: the top-k router and the row lists that turn "token t uses experts ids[t, :]" into
// one contiguous row segment per expert, which the grouped product of gemm_any.cu walks.  The expert products themselves
// are matrix products (gemm_any.cu); the weighted sum of their outputs is part of the sublayer's tail (resid_tail_kernel).
//
// Router arithmetic is fp32 throughout: logits + bias, selection, and the weights of the selected experts: the softmax over
// the selected logits only (MOE_W_SOFTMAX), each one's own sigmoid (MOE_W_SIGMOID; the order of sigmoid scores is the order
// of the logits), or the selected ones' shares of a softmax over all of them (MOE_W_SHARE; the bias then enters the choice, after
// the softmax, and not the weights).
#include <cfloat>

#include "kernels.h"
#include "launch.cuh"
#include "ptx.cuh"

namespace tgis {
namespace {

constexpr int ROUTE_WARPS = 4;

// one warp per token; dynamic shared memory: ROUTE_WARPS x (E + groups) floats
__global__ void __launch_bounds__(ROUTE_WARPS * 32)
moe_route_kernel(const float* __restrict__ logits, int ld, const float* __restrict__ bias, int E, int top,
                 int32_t* __restrict__ ids, float* __restrict__ w, float* __restrict__ side_gate, int T, int weight_mode, int groups, int keep) {
  extern __shared__ float sm[];
  griddep_launch();
  griddep_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * ROUTE_WARPS + warp;
  if (t >= T) return;
  float* z = sm + (size_t)warp * (E + groups);
  const float* row = logits + (size_t)t * ld;
  float z_max = 0.f, z_sum = 1.f;   // MOE_W_SHARE: the softmax over all logits
  if (weight_mode == MOE_W_SHARE) {
    z_max = -FLT_MAX;
    for (int e = lane; e < E; e += 32) z_max = fmaxf(z_max, row[e]);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) z_max = fmaxf(z_max, __shfl_xor_sync(0xffffffffu, z_max, o));
    z_sum = 0.f;
    for (int e = lane; e < E; e += 32) z_sum += expf(row[e] - z_max);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) z_sum += __shfl_xor_sync(0xffffffffu, z_sum, o);
  }
  for (int e = lane; e < E; e += 32)
    z[e] = (weight_mode == MOE_W_SHARE ? expf(row[e] - z_max) / z_sum : row[e]) + (bias ? bias[e] : 0.f);
  if (side_gate != nullptr && lane == 0) side_gate[t] = 1.f / (1.f + expf(-row[E]));
  __syncwarp();
  if (groups > 1) {   // members of all but the `keep` best groups are out of the choice
    const int per = E / groups;
    float* gs = z + E;
    for (int g = lane; g < groups; g += 32) {
      float m = -FLT_MAX;
      for (int e = g * per; e < (g + 1) * per; ++e) m = fmaxf(m, z[e]);
      gs[g] = m;
    }
    __syncwarp();
    for (int e = lane; e < E; e += 32) {
      const int g = e / per;
      int better = 0;   // groups that come before this one
      for (int o = 0; o < groups; ++o) better += (gs[o] > gs[g] || (gs[o] == gs[g] && o < g)) ? 1 : 0;
      if (better >= keep) z[e] = -FLT_MAX;
    }
    __syncwarp();
  }
  float my_val = -FLT_MAX;  // lane k keeps the k-th selected logit
  int my_id = 0;
  for (int k = 0; k < top; ++k) {
    float best = -FLT_MAX;
    int bi = 0x7fffffff;
    for (int e = lane; e < E; e += 32) {
      const float v = z[e];
      if (v > best || (v == best && e < bi)) { best = v; bi = e; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
    }
    if (lane == (k & 31)) { my_val = best; my_id = bi; }
    if (lane == 0) {
      ids[(size_t)t * top + k] = bi;
      z[bi] = -FLT_MAX;
    }
    __syncwarp();
  }
  if (weight_mode == MOE_W_SIGMOID) {   // every chosen expert weighs its own sigmoid score; nothing is renormalised
    if (lane < top) w[(size_t)t * top + lane] = 1.f / (1.f + expf(-my_val));
    return;
  }
  if (weight_mode == MOE_W_SHARE) {   // the chosen scores (without the bias) over their sum
    const float s = lane < top ? expf(row[my_id] - z_max) / z_sum : 0.f;
    float tot = s;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) tot += __shfl_xor_sync(0xffffffffu, tot, o);
    if (lane < top) w[(size_t)t * top + lane] = s / (tot + 1e-20f);
    return;
  }
  // softmax over the selected logits (the first selected one is the largest)
  const float m = __shfl_sync(0xffffffffu, my_val, 0);
  float e = lane < top ? expf(my_val - m) : 0.f;
  float sum = e;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
  if (lane < top) w[(size_t)t * top + lane] = e / sum;
}

// single CTA; dynamic shared memory: 2 E ints
__global__ void __launch_bounds__(1024)
moe_align_kernel(const int32_t* __restrict__ ids, int n, int E, int32_t* __restrict__ seg_off, int32_t* __restrict__ order,
                 int32_t* __restrict__ inv) {
  extern __shared__ int sm_i[];
  int* cnt = sm_i;
  int* cur = sm_i + E;
  griddep_launch();
  griddep_wait();
  for (int e = threadIdx.x; e < E; e += blockDim.x) cnt[e] = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < n; i += blockDim.x) atomicAdd(&cnt[ids[i]], 1);
  __syncthreads();
  if (threadIdx.x == 0) {
    int run = 0;
    for (int e = 0; e < E; ++e) {
      seg_off[e] = run;
      cur[e] = run;
      run += cnt[e];
    }
    seg_off[E] = run;
  }
  __syncthreads();
  // the place of a row inside its segment does not enter any result (every row of a grouped product is computed alone)
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const int p = atomicAdd(&cur[ids[i]], 1);
    order[p] = i;
    inv[i] = p;
  }
}

// one CTA per layer; dynamic shared memory: 2 max_E ints
__global__ void __launch_bounds__(1024)
moe_table_align_kernel(const MoeTable* __restrict__ layers, const int32_t* __restrict__ tok, int vocab, int T) {
  extern __shared__ int sm_i[];
  griddep_launch();
  griddep_wait();
  const MoeTable a = layers[blockIdx.x];
  const int E = a.E, top = a.top, n = T * top, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  int* cnt = sm_i;
  int* cur = sm_i + E;
  __shared__ int warp_tot[32];
  auto expert = [&](int i) {
    const int t = tok[i / top];
    return a.table[(size_t)(t >= 0 && t < vocab ? t : 0) * top + i % top];   // (as the embedding reads ids outside the vocabulary)
  };
  for (int e = threadIdx.x; e < E; e += 1024) cnt[e] = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < n; i += 1024) atomicAdd(&cnt[expert(i)], 1);
  __syncthreads();
  int base = 0;   // exclusive prefix sum, 1024 experts at a time
  for (int e0 = 0; e0 < E; e0 += 1024) {
    const int e = e0 + threadIdx.x, c = e < E ? cnt[e] : 0;
    int run = c;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int up = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += up;
    }
    if (lane == 31) warp_tot[warp] = run;
    __syncthreads();
    int before = base, all = 0;
    for (int w = 0; w < 32; ++w) {
      if (w < warp) before += warp_tot[w];
      all += warp_tot[w];
    }
    if (e < E) {
      cur[e] = before + run - c;
      a.seg_off[e] = before + run - c;
    }
    base += all;
    __syncthreads();
  }
  if (threadIdx.x == 0) a.seg_off[E] = base;
  // the place of a row inside its segment does not enter any result (every row of a grouped product is computed alone)
  for (int i = threadIdx.x; i < n; i += 1024) {
    const int p = atomicAdd(&cur[expert(i)], 1);
    a.order[p] = i;
    a.inv[i] = p;
  }
}

}  // namespace

cudaError_t moe_table_align_launch(const MoeTable* layers_dev, int n_layers, int max_E, const int32_t* tok, int vocab, int T, cudaStream_t stream) {
  if (T <= 0 || n_layers <= 0) return cudaSuccess;
  if (max_E < 1 || (size_t)2 * max_E * 4 > 40 * 1024) return cudaErrorInvalidValue;
  return launch_k(moe_table_align_kernel, dim3(n_layers), dim3(1024), (size_t)2 * max_E * sizeof(int), stream, layers_dev, tok, vocab, T);
}

cudaError_t moe_route_launch(const float* logits, int ld, const float* bias, int E, int top, int32_t* ids, float* w,
                             float* side_gate, int T, cudaStream_t stream, int weight_mode, int groups, int keep) {
  if (T <= 0) return cudaSuccess;
  if (groups < 1 || E % groups != 0 || keep < 1 || keep > groups) return cudaErrorInvalidValue;
  if (top < 1 || top > 32 || top > E / groups * keep || (size_t)ROUTE_WARPS * (E + groups) * 4 > 48 * 1024) return cudaErrorInvalidValue;
  return launch_k(moe_route_kernel, dim3((T + ROUTE_WARPS - 1) / ROUTE_WARPS), dim3(ROUTE_WARPS * 32),
                  (size_t)ROUTE_WARPS * (E + groups) * sizeof(float), stream, logits, ld, bias, E, top, ids, w, side_gate, T, weight_mode,
                  groups, keep);
}

cudaError_t moe_align_launch(const int32_t* ids, int T, int top, int E, int32_t* seg_off, int32_t* order, int32_t* inv,
                             cudaStream_t stream) {
  if (T <= 0) return cudaSuccess;
  if ((size_t)2 * E * 4 > 48 * 1024) return cudaErrorInvalidValue;
  return launch_k(moe_align_kernel, dim3(1), dim3(1024), (size_t)2 * E * sizeof(int), stream, ids, T * top, E, seg_off, order,
                  inv);
}

}  // namespace tgis
