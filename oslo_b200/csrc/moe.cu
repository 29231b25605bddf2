// Mixture-of-experts feed-forward: routing, the plan that turns (token, choice) pairs into expert-contiguous rows, and the
// expert products that do not go through the tcgen05 grouped GEMM (oslo_gemm_grouped, gemm_sm100.cu).
//
//   route:   z = W_router h + b (32-bit), the `top` largest, softmax over those only; or scored: s = softmax(W_router h) over
//            all outputs, the `top` largest s + b, weights s / sum of the chosen s. Outputs past the experts stand for the
//            input itself: no slot and no product, the step that joins the residual stream knows them. Or sigmoid scores: the
//            `top` largest z, weights sigmoid(z)
//   prefill: moe_plan assigns every (token, choice) a slot; an expert's slots are consecutive and start at a multiple of
//            128, so a 128-row tile of the grouped GEMM belongs to one expert (tile_group); moe_gather copies the rows.
//            Everything stays on the device: no counts are read back, grids are sized for the worst case. Units: relu^2,
//            or silu(gate) * up or its clamped form with the rows of the two matrices in turns, so that a pair of columns is one
//            output. Where a token's weight belongs to what the expert reads, it goes in with the copy.
//   decode:  a few rows: one warp per output element of the chosen experts, straight from the expert's weights.
// The down projection leaves one row per slot; the residual join adds them up with their weights.
#include <cooperative_groups.h>
#include <math_constants.h>

#include <algorithm>

#include "num.cuh"
#include "oslo_kernels.h"

namespace cg = cooperative_groups;

namespace oslo {

constexpr int MOE_TILE = 128;          // rows per grouped-GEMM tile
constexpr int MOE_MAX_EXPERTS = 2048;

enum { ROUTE_CHOSEN = 0, ROUTE_SCORED = 1, ROUTE_SIGMOID = 2 };   // softmax over the chosen; over all; sigmoids

// the `top` largest of z[0..E) (shared memory, overwritten), ties to the lower index; softmax over them, or (sig) the sigmoid
// of each. One warp.
__device__ __forceinline__ void pick_top(float* z, int E, int top, int* idx, float* wgt, int lane, bool sig) {
  float first = 0.f, sum = 0.f;
  for (int j = 0; j < top; ++j) {
    float best = -CUDART_INF_F;
    int at = E;
    for (int e = lane; e < E; e += 32) {
      const float v = z[e];
      if (v > best || (at == E && v == best)) { best = v; at = e; }
    }
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, off);
      const int oa = __shfl_xor_sync(0xffffffffu, at, off);
      if (ov > best || (ov == best && oa < at)) { best = ov; at = oa; }
    }
    if (at >= E) { at = 0; best = 0.f; }               // only NaN logits get here
    if (j == 0) first = best;
    const float ex = sig ? 1.0f / (1.0f + expf(-best)) : expf(best - first);
    sum += ex;
    if (lane == 0) {
      idx[j] = at;
      wgt[j] = ex;
      z[at] = -CUDART_INF_F;
    }
    __syncwarp();
  }
  if (lane == 0 && !sig) {
    const float inv = 1.0f / sum;
    for (int j = 0; j < top; ++j) wgt[j] *= inv;
  }
}

// z[0..E) become scores, the softmax over all of them; the `top` largest score + b, ties to the lower index; weights: the chosen
// scores divided by their sum. `ch` [E] is work space. One warp.
template <typename T>
__device__ __forceinline__ void pick_scored(float* z, float* ch, const T* b, int E, int top, int* idx, float* wgt, int lane) {
  float mx = -CUDART_INF_F;
  for (int e = lane; e < E; e += 32) mx = fmaxf(mx, z[e]);
#pragma unroll
  for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
  float sum = 0.f;
  for (int e = lane; e < E; e += 32) {
    z[e] = expf(z[e] - mx);
    sum += z[e];
  }
  sum = warp_sum(sum);
  for (int e = lane; e < E; e += 32) {
    z[e] = z[e] / sum;
    ch[e] = z[e] + Num<T>::to(b[e]);
  }
  __syncwarp();
  float tot = 0.f;
  for (int j = 0; j < top; ++j) {
    float best = -CUDART_INF_F;
    int at = E;
    for (int e = lane; e < E; e += 32) {
      const float v = ch[e];
      if (v > best || (at == E && v == best)) { best = v; at = e; }
    }
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, off);
      const int oa = __shfl_xor_sync(0xffffffffu, at, off);
      if (ov > best || (ov == best && oa < at)) { best = ov; at = oa; }
    }
    if (at >= E) at = 0;                               // only NaN logits get here
    const float s = z[at];
    tot += s;
    if (lane == 0) {
      idx[j] = at;
      wgt[j] = s;
    }
    __syncwarp();
    if (lane == 0) ch[at] = -CUDART_INF_F;
    __syncwarp();
  }
  if (lane == 0) {
    const float inv = 1.0f / (tot + 1e-20f);
    for (int j = 0; j < top; ++j) wgt[j] *= inv;
  }
}

// logits from the kernel itself: a cluster of RT_CLUSTER blocks per row shares the experts, the first block collects the
// logits over distributed shared memory and picks
constexpr int RT_CLUSTER = 8;
template <typename T, int VEC>
__global__ void __cluster_dims__(RT_CLUSTER, 1, 1) __launch_bounds__(256)
route_kernel(const T* __restrict__ h, long long ldh, const T* __restrict__ w, const T* __restrict__ bias, int* __restrict__ idx,
             float* __restrict__ wgt, int E, int K, int top, int scored) {
  extern __shared__ float z[];         // [E] (ROUTE_SCORED: and [E] of work space), used in the first block
  cg::cluster_group cluster = cg::this_cluster();
  const int rank = static_cast<int>(cluster.block_rank());
  float* z0 = cluster.map_shared_rank(z, 0);
  const long long row = blockIdx.y;
  const T* x = h + row * ldh;
  const int lane = threadIdx.x & 31;
  for (int e = rank + RT_CLUSTER * (threadIdx.x >> 5); e < E; e += RT_CLUSTER * (blockDim.x >> 5)) {
    const T* we = w + static_cast<long long>(e) * K;
    float acc = 0.f;
#pragma unroll 8
    for (int k = lane * VEC; k < K; k += 32 * VEC) {
      float a[VEC], b[VEC];
      load_vec<T, VEC>(we + k, a);
      load_vec<T, VEC>(x + k, b);
#pragma unroll
      for (int i = 0; i < VEC; ++i) acc = fmaf(a[i], b[i], acc);
    }
    acc = warp_sum(acc);
    if (lane == 0) z0[e] = bias == nullptr || scored == ROUTE_SCORED ? acc : acc + Num<T>::to(bias[e]);
  }
  cluster.sync();                      // also keeps the first block's shared memory alive until all have written
  if (rank == 0 && threadIdx.x < 32) {
    if (scored == ROUTE_SCORED) pick_scored<T>(z, z + E, bias, E, top, idx + row * top, wgt + row * top, lane);
    else pick_top(z, E, top, idx + row * top, wgt + row * top, lane, scored == ROUTE_SIGMOID);
  }
}

// logits [rows, E] (32-bit, without the bias, rows ldl apart) from a GEMM: one warp per row
template <typename T>
__global__ void __launch_bounds__(128) route_logits_kernel(const float* __restrict__ logits, long long ldl, const T* __restrict__ bias,
                                                           int* __restrict__ idx, float* __restrict__ wgt, long long rows,
                                                           int E, int top, int scored) {
  extern __shared__ float rl_smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long row = static_cast<long long>(blockIdx.x) * 4 + warp;
  if (row >= rows) return;
  float* z = rl_smem + warp * E * (scored == ROUTE_SCORED ? 2 : 1);
  const bool add = bias != nullptr && scored != ROUTE_SCORED;
  for (int e = lane; e < E; e += 32) z[e] = add ? logits[row * ldl + e] + Num<T>::to(bias[e]) : logits[row * ldl + e];
  __syncwarp();
  if (scored == ROUTE_SCORED) pick_scored<T>(z, z + E, bias, E, top, idx + row * top, wgt + row * top, lane);
  else pick_top(z, E, top, idx + row * top, wgt + row * top, lane, scored == ROUTE_SIGMOID);
}

// counts per expert -> start slot of every expert (multiple of MOE_TILE), expert of every tile, number of tiles
__global__ void __launch_bounds__(1024) moe_plan_kernel(const int* __restrict__ idx, long long pairs, int E,
                                                        int* __restrict__ cursor, int* __restrict__ tile_group,
                                                        int* __restrict__ n_tiles, int max_tiles) {
  __shared__ int count[MOE_MAX_EXPERTS];
  __shared__ int start[MOE_MAX_EXPERTS];
  __shared__ int total;
  for (int e = threadIdx.x; e < E; e += blockDim.x) count[e] = 0;
  __syncthreads();
  for (long long i = threadIdx.x; i < pairs; i += blockDim.x)
    if (idx[i] < E) atomicAdd(&count[idx[i]], 1);      // the others are no experts
  __syncthreads();
  if (threadIdx.x == 0) {
    int t = 0;
    for (int e = 0; e < E; ++e) {
      start[e] = t;
      t += (count[e] + MOE_TILE - 1) / MOE_TILE;
    }
    total = min(t, max_tiles);
    *n_tiles = total;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x) {
    cursor[e] = start[e] * MOE_TILE;
    const int n = (count[e] + MOE_TILE - 1) / MOE_TILE;
    for (int i = 0; i < n; ++i)
      if (start[e] + i < max_tiles) tile_group[start[e] + i] = e;
  }
}

// one block per (token, choice): take the next slot of its expert and copy the token's row there, times `scale` [pairs] if given
template <typename T, int VEC>
__global__ void __launch_bounds__(128) moe_gather_kernel(const T* __restrict__ h, long long ldh, const int* __restrict__ idx,
                                                         int* __restrict__ cursor, int* __restrict__ slots, T* __restrict__ out,
                                                         const float* __restrict__ scale, int K, int top, int max_slots, int E) {
  __shared__ int slot_s;
  const long long pair = blockIdx.x;
  if (idx[pair] >= E) {                                // no expert, no slot
    if (threadIdx.x == 0) slots[pair] = -1;
    return;
  }
  if (threadIdx.x == 0) {
    slot_s = atomicAdd(&cursor[idx[pair]], 1);
    slots[pair] = slot_s;
  }
  __syncthreads();
  const int slot = slot_s;
  if (slot >= max_slots) return;
  const T* src = h + pair / top * ldh;
  T* dst = out + static_cast<long long>(slot) * K;
  if (scale != nullptr) {
    const float f = scale[pair];
    for (int k = threadIdx.x * VEC; k < K; k += blockDim.x * VEC) {
      float v[VEC];
      load_vec<T, VEC>(src + k, v);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] *= f;
      store_vec<T, VEC>(dst + k, v);
    }
    return;
  }
  for (int k = threadIdx.x * VEC; k < K; k += blockDim.x * VEC)
    *reinterpret_cast<Pack<T, VEC>*>(dst + k) = *reinterpret_cast<const Pack<T, VEC>*>(src + k);
}

// GLU, CLAMPED: columns in pairs (gate, up), half as many outputs
enum { UNIT_NONE = 0, UNIT_RELU2 = 1, UNIT_GLU = 2, UNIT_CLAMPED = 3 };
__device__ __forceinline__ float pair_unit(float g, float u, int unit, float limit, float alpha) {
  if (unit == UNIT_GLU) return silu_f(g) * u;
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g * sigmoid_f(alpha * g) * (u + 1.0f);
}

// scalar grouped product for types and sizes outside the tensor-core path: 32 x 64 outputs per block
template <typename T>
__global__ void __launch_bounds__(256) moe_grouped_kernel(const T* __restrict__ a, const T* __restrict__ w, T* __restrict__ out,
                                                          const int* __restrict__ tile_group, const int* __restrict__ n_tiles,
                                                          int N, int K, int unit, float limit, float alpha) {
  constexpr int BMS = 32, BNS = 64, BKS = 16;
  __shared__ float as[BKS][BMS + 1];
  __shared__ float bs[BKS][BNS + 1];
  const int m0 = blockIdx.y * BMS, n0 = blockIdx.x * BNS;
  const int tile = m0 / MOE_TILE;
  if (tile >= *n_tiles) return;
  const T* b = w + static_cast<long long>(tile_group[tile]) * N * K;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[2][4] = {};
  for (int k0 = 0; k0 < K; k0 += BKS) {
    for (int e = threadIdx.x; e < BMS * BKS; e += 256) {
      const int r = e / BKS, k = e % BKS;
      as[k][r] = k0 + k < K ? Num<T>::to(a[static_cast<long long>(m0 + r) * K + k0 + k]) : 0.f;
    }
    for (int e = threadIdx.x; e < BNS * BKS; e += 256) {
      const int r = e / BKS, k = e % BKS;
      bs[k][r] = (k0 + k < K && n0 + r < N) ? Num<T>::to(b[static_cast<long long>(n0 + r) * K + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < BKS; ++k) {
      const float a0 = as[k][ty * 2], a1 = as[k][ty * 2 + 1];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float x = bs[k][tx + 16 * j];
        acc[0][j] = fmaf(a0, x, acc[0][j]);
        acc[1][j] = fmaf(a1, x, acc[1][j]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx + 16 * j;
      float v = acc[i][j];
      if (unit >= UNIT_GLU) {                          // N is even: a pair of columns is in one pair of lanes
        const float up = __shfl_xor_sync(0xffffffffu, v, 1);
        if (n < N && (n & 1) == 0)
          out[static_cast<long long>(m0 + ty * 2 + i) * (N / 2) + n / 2] = Num<T>::from(pair_unit(v, up, unit, limit, alpha));
        continue;
      }
      if (n >= N) continue;
      if (unit == UNIT_RELU2) { v = fmaxf(v, 0.f); v *= v; }
      out[static_cast<long long>(m0 + ty * 2 + i) * N + n] = Num<T>::from(v);
    }
}

// few rows: out[pair, n] = act(w[idx[pair]][n, :] . x[row of pair, :] * scale[pair]); groups of `wg` warps share the k range of 4 outputs
// and walk over the output groups, so that the chosen expert is looked up once per block
template <typename T, int VEC>
__global__ void __launch_bounds__(256, 4) moe_few_kernel(const T* __restrict__ x, long long ldx, const int* __restrict__ idx,
                                                         const T* __restrict__ w, T* __restrict__ out, int N, int K,
                                                         int per_row, int unit, int wg, int E, float limit, float alpha,
                                                         const float* __restrict__ scale) {
  __shared__ float red[2][8][4];
  if (idx[blockIdx.y] >= E) return;                    // no expert: nobody reads the row
  const int pair = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* src = x + static_cast<long long>(pair / per_row) * ldx;
  const T* we = w + static_cast<long long>(idx[pair]) * N * K;
  const int group = warp / wg, gw = warp % wg, per_block = 8 / wg * 4;
  for (int nb = blockIdx.x * per_block, it = 0; nb < N; nb += gridDim.x * per_block, ++it) {
    const int n0 = nb + group * 4, nn = min(4, N - n0);      // nn may be <= 0 for the last groups
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int k = (gw * 32 + lane) * VEC; k < K; k += wg * 32 * VEC) {
      Pack<T, VEC> v[4];
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (j < nn) v[j] = *reinterpret_cast<const Pack<T, VEC>*>(we + static_cast<long long>(n0 + j) * K + k);
      float xv[VEC];
      load_vec<T, VEC>(src + k, xv);
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (j < nn) {
#pragma unroll
          for (int i = 0; i < VEC; ++i) acc[j] = fmaf(Num<T>::to(v[j].e[i]), xv[i], acc[j]);
        }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[j] = warp_sum(acc[j]);
    float(*r)[4] = red[it & 1];
    if (lane == 0) {
#pragma unroll
      for (int j = 0; j < 4; ++j) r[warp][j] = acc[j];
    }
    __syncthreads();                   // the other half of `red` is free again: it was read before this barrier
    if (gw == 0) {                     // uniform over the warp
      float s = 0.f;
      if (lane < nn)
        for (int g = 0; g < wg; ++g) s += r[warp + g][lane];
      if (scale != nullptr) s *= scale[pair];
      if (unit >= UNIT_GLU) {
        const float up = __shfl_xor_sync(0xffffffffu, s, 1);
        if (lane < nn && (lane & 1) == 0)
          out[static_cast<long long>(pair) * (N / 2) + (n0 + lane) / 2] = Num<T>::from(pair_unit(s, up, unit, limit, alpha));
      } else if (lane < nn) {
        if (unit == UNIT_RELU2) { s = fmaxf(s, 0.f); s *= s; }
        out[static_cast<long long>(pair) * N + n0 + lane] = Num<T>::from(s);
      }
    }
  }
}

}  // namespace oslo

extern "C" int oslo_moe_route(const void* h, long long ldh, const void* w, const void* bias, const float* logits, long long ldl,
                              int* idx, float* wgt, long long rows, int E, int K, int top, int scored, int dtype, cudaStream_t stream) {
  using namespace oslo;
  const size_t per_row = (scored == ROUTE_SCORED ? 2 : 1) * E * sizeof(float);
  if (rows <= 0) return 0;
  if (E <= 0 || E > MOE_MAX_EXPERTS || top <= 0 || top > E || rows > 0x7fffffffll) return -1;
  if (scored < ROUTE_CHOSEN || scored > ROUTE_SIGMOID || (scored == ROUTE_SCORED && bias == nullptr)) return -1;
  const size_t te = dtype == OSLO_DT_FP32 ? 4 : 2;
  if (logits) {
    OSLO_DISPATCH_T(dtype, {
      route_logits_kernel<T><<<static_cast<unsigned>((rows + 3) / 4), 128, 4 * per_row, stream>>>(
          logits, ldl, static_cast<const T*>(bias), idx, wgt, rows, E, top, scored);
    });
    return static_cast<int>(cudaGetLastError());
  }
  if (rows > 65535) return -1;         // larger batches bring their logits
  const int v = static_cast<int>(16 / te);
  const bool vec = K % v == 0 && ldh % v == 0 && aligned_to(w, 16) && aligned_to(h, 16);
  const dim3 grid(RT_CLUSTER, static_cast<unsigned>(rows));
  OSLO_DISPATCH_T(dtype, {
    constexpr int V = 16 / sizeof(T);
    if (vec)
      route_kernel<T, V><<<grid, 256, per_row, stream>>>(static_cast<const T*>(h), ldh, static_cast<const T*>(w),
                                                                   static_cast<const T*>(bias), idx, wgt, E, K, top, scored);
    else
      route_kernel<T, 1><<<grid, 256, per_row, stream>>>(static_cast<const T*>(h), ldh, static_cast<const T*>(w),
                                                                   static_cast<const T*>(bias), idx, wgt, E, K, top, scored);
  });
  return static_cast<int>(cudaGetLastError());
}

extern "C" int oslo_moe_plan(const void* h, long long ldh, const int* idx, int* cursor, int* tile_group, int* n_tiles, int* slots,
                             void* rows_out, const float* scale, long long pairs, int E, int K, int top, int max_tiles, int dtype,
                             cudaStream_t stream) {
  using namespace oslo;
  if (pairs <= 0) return 0;
  if (E <= 0 || E > MOE_MAX_EXPERTS || pairs > 0x7fffffffll) return -1;
  const size_t te = dtype == OSLO_DT_FP32 ? 4 : 2;
  moe_plan_kernel<<<1, 1024, 0, stream>>>(idx, pairs, E, cursor, tile_group, n_tiles, max_tiles);
  const int v = static_cast<int>(16 / te);
  const bool vec = K % v == 0 && ldh % v == 0 && aligned_to(h, 16) && aligned_to(rows_out, 16);
  OSLO_DISPATCH_T(dtype, {
    constexpr int V = 16 / sizeof(T);
    if (vec)
      moe_gather_kernel<T, V><<<static_cast<unsigned>(pairs), 128, 0, stream>>>(
          static_cast<const T*>(h), ldh, idx, cursor, slots, static_cast<T*>(rows_out), scale, K, top, max_tiles * MOE_TILE, E);
    else
      moe_gather_kernel<T, 1><<<static_cast<unsigned>(pairs), 128, 0, stream>>>(
          static_cast<const T*>(h), ldh, idx, cursor, slots, static_cast<T*>(rows_out), scale, K, top, max_tiles * MOE_TILE, E);
  });
  return static_cast<int>(cudaGetLastError());
}

extern "C" int oslo_moe_grouped(const void* a, const void* w, void* out, const int* tile_group, const int* n_tiles,
                                int max_tiles, int N, int K, int unit, float limit, float alpha, int dtype, cudaStream_t stream) {
  using namespace oslo;
  if (max_tiles <= 0 || N <= 0) return 0;
  if (unit >= UNIT_GLU && N % 2) return -1;
  if (static_cast<long long>(max_tiles) * (MOE_TILE / 32) > 65535) return -1;
  OSLO_DISPATCH_T(dtype, {
    moe_grouped_kernel<T><<<dim3((N + 63) / 64, max_tiles * (MOE_TILE / 32)), 256, 0, stream>>>(
        static_cast<const T*>(a), static_cast<const T*>(w), static_cast<T*>(out), tile_group, n_tiles, N, K, unit, limit, alpha);
  });
  return static_cast<int>(cudaGetLastError());
}

extern "C" int oslo_moe_few(const void* x, long long ldx, const int* idx, const void* w, void* out, int pairs, int per_row,
                            int N, int K, int unit, float limit, float alpha, const float* scale, int E, int dtype,
                            cudaStream_t stream) {
  using namespace oslo;
  if (pairs <= 0 || N <= 0) return 0;
  if (pairs > 65535 || per_row < 1 || (unit >= UNIT_GLU && N % 2)) return -1;
  const size_t te = dtype == OSLO_DT_FP32 ? 4 : 2;
  const int v = static_cast<int>(16 / te);
  const bool vec = K % v == 0 && ldx % v == 0 && aligned_to(w, 16) && aligned_to(x, 16);
  int wg = 8;                          // warps on one output group: at least one full stride each
  while (wg > 1 && K < wg * 32 * (vec ? v : 1)) wg /= 2;
  const int per_block = 8 / wg * 4;
  const int want = (148 * 4 + pairs - 1) / pairs;
  const dim3 grid(std::min((N + per_block - 1) / per_block, want), pairs);
  OSLO_DISPATCH_T(dtype, {
    constexpr int V = 16 / sizeof(T);
    if (vec)
      moe_few_kernel<T, V><<<grid, 256, 0, stream>>>(static_cast<const T*>(x), ldx, idx, static_cast<const T*>(w),
                                                     static_cast<T*>(out), N, K, per_row, unit, wg, E, limit, alpha, scale);
    else
      moe_few_kernel<T, 1><<<grid, 256, 0, stream>>>(static_cast<const T*>(x), ldx, idx, static_cast<const T*>(w),
                                                     static_cast<T*>(out), N, K, per_row, unit, wg, E, limit, alpha, scale);
  });
  return static_cast<int>(cudaGetLastError());
}
