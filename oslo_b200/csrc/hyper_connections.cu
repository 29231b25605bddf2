// Residual streams with hyper-connections: the step between two sublayers, one pass over the rows in 32-bit.
//
//   y    = the sublayer's result: one row per token, or the weighted sum of the rows a mixture of experts left in its slot
//          buffer (choices that are no expert stand for the sublayer's input), plus a shared expert's row times the sigmoid
//          of its gate
//   x_t <- sum_s mix[s, t] x_s + out[t] y                 every stream from the old ones
//   u    = sum_t in[t] x_t                                what the next sublayer reads (in null: the plain sum)
//   h    = u / sqrt(mean(u^2) + eps) * (1 + w) * scale
// Without a result the streams stay and only h is written. A stream stride of 0 stands for streams that are all equal.
#include <algorithm>

#include "num.cuh"
#include "oslo_kernels.h"

namespace oslo {

constexpr int HYPER_MAX_TOP = 64;

struct HyperParams {
  const float* x; long long x_row, x_stream;   // element strides of rows and streams
  const void* y; long long ldy;                // nullptr: no result
  const int* slots;                            // [rows, top] rows of y, or nullptr: row * top + j
  const float* weights;                        // [rows, top], or nullptr: y has one row per token
  const int* choice; int experts;              // [rows, top]: choices >= experts stand for own; or nullptr
  const void* own; long long ld_own;
  const void* shared; long long ld_shared;     // or nullptr
  const void* gate; long long ld_gate;
  const void *w_out, *mix, *w_in, *w_norm;     // [n], [n, n] from x to, [n] or nullptr, [cols]
  float* x_out;                                // [rows, n, cols]
  void* h;
  int n, top, cols;
  float eps, scale;
};

// NS: streams kept in registers, n <= NS
template <typename T, int VEC, int NS>
__global__ void __launch_bounds__(256) hyper_join_kernel(const HyperParams p) {
  extern __shared__ float row_s[];             // [cols]
  __shared__ float red[32], mix[NS][NS], w_out[NS], w_in[NS], wgt[HYPER_MAX_TOP];
  __shared__ const T* src[HYPER_MAX_TOP];
  const long long row = blockIdx.x;
  const int n = p.n;
  const bool joins = p.y != nullptr;
  for (int e = threadIdx.x; e < NS * NS; e += blockDim.x) {
    const int s = e / NS, t = e % NS;
    mix[s][t] = joins && s < n && t < n ? Num<T>::to(static_cast<const T*>(p.mix)[s * n + t]) : 0.f;
  }
  for (int t = threadIdx.x; t < NS; t += blockDim.x) {
    w_out[t] = joins && t < n ? Num<T>::to(static_cast<const T*>(p.w_out)[t]) : 0.f;
    w_in[t] = t < n ? (p.w_in ? Num<T>::to(static_cast<const T*>(p.w_in)[t]) : 1.f) : 0.f;
  }
  const T* y = static_cast<const T*>(p.y);
  if (p.weights != nullptr) {
    for (int j = threadIdx.x; j < p.top; j += blockDim.x) {
      const long long at = row * p.top + j;
      wgt[j] = p.weights[at];
      if (p.choice != nullptr && p.choice[at] >= p.experts) src[j] = static_cast<const T*>(p.own) + row * p.ld_own;
      else src[j] = y + (p.slots ? static_cast<long long>(p.slots[at]) : at) * p.ldy;
    }
  }
  __syncthreads();
  const float shared_w = p.shared ? sigmoid_f(Num<T>::to(static_cast<const T*>(p.gate)[row * p.ld_gate])) : 0.f;
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < p.cols; c += blockDim.x * VEC) {
    float v[VEC], x[NS][VEC], u[VEC];
#pragma unroll
    for (int s = 0; s < NS; ++s)
      if (s < n) {
        load_vec<float, VEC>(p.x + row * p.x_row + s * p.x_stream + c, x[s]);
      } else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) x[s][i] = 0.f;
      }
#pragma unroll
    for (int i = 0; i < VEC; ++i) u[i] = 0.f;
    if (joins) {
      if (p.weights == nullptr) {
        load_vec<T, VEC>(y + row * p.ldy + c, v);
      } else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = 0.f;
#pragma unroll 4
        for (int j = 0; j < p.top; ++j) {
          float e[VEC];
          load_vec<T, VEC>(src[j] + c, e);
#pragma unroll
          for (int i = 0; i < VEC; ++i) v[i] = fmaf(wgt[j], e[i], v[i]);
        }
      }
      if (p.shared != nullptr) {
        float e[VEC];
        load_vec<T, VEC>(static_cast<const T*>(p.shared) + row * p.ld_shared + c, e);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = fmaf(shared_w, e[i], v[i]);
      }
#pragma unroll
      for (int t = 0; t < NS; ++t) {
        if (t >= n) break;
        float o[VEC];
#pragma unroll
        for (int i = 0; i < VEC; ++i) o[i] = w_out[t] * v[i];
#pragma unroll
        for (int s = 0; s < NS; ++s)
#pragma unroll
          for (int i = 0; i < VEC; ++i) o[i] = fmaf(mix[s][t], x[s][i], o[i]);
        store_vec<float, VEC>(p.x_out + (row * n + t) * p.cols + c, o);
#pragma unroll
        for (int i = 0; i < VEC; ++i) u[i] = fmaf(w_in[t], o[i], u[i]);
      }
    } else {
#pragma unroll
      for (int s = 0; s < NS; ++s)
#pragma unroll
        for (int i = 0; i < VEC; ++i) u[i] = fmaf(w_in[s], x[s][i], u[i]);
    }
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      ss = fmaf(u[i], u[i], ss);
      row_s[c + i] = u[i];
    }
  }
  ss = block_sum(ss, red);
  const float r = p.scale / sqrtf(ss / p.cols + p.eps);
  for (int c = threadIdx.x * VEC; c < p.cols; c += blockDim.x * VEC) {   // every thread revisits its own elements
    float v[VEC], w[VEC];
    load_vec<T, VEC>(static_cast<const T*>(p.w_norm) + c, w);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = row_s[c + i] * r * (1.0f + w[i]);
    store_vec<T, VEC>(static_cast<T*>(p.h) + row * p.cols + c, v);
  }
}

template <typename T, int VEC, int NS>
static int hyper_launch(const HyperParams& p, long long rows, cudaStream_t st) {
  const size_t smem = static_cast<size_t>(p.cols) * sizeof(float);
  if (smem > 200 * 1024) return -3;
  if (smem > 40 * 1024) {                      // static arrays come on top
    cudaError_t e = cudaFuncSetAttribute(hyper_join_kernel<T, VEC, NS>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  const int threads = p.cols >= 1024 ? 256 : (p.cols >= 512 ? 128 : 64);
  hyper_join_kernel<T, VEC, NS><<<static_cast<unsigned>(rows), threads, smem, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}
template <typename T, int VEC>
static int hyper_dispatch(const HyperParams& p, long long rows, cudaStream_t st) {
  if (p.n <= 2) return hyper_launch<T, VEC, 2>(p, rows, st);
  if (p.n <= 4) return hyper_launch<T, VEC, 4>(p, rows, st);
  if (p.n <= 8) return hyper_launch<T, VEC, 8>(p, rows, st);
  if (p.n <= 16) return hyper_launch<T, 1, 16>(p, rows, st);
  return -3;
}

}  // namespace oslo

extern "C" int oslo_hyper_join(const float* x, long long x_row, long long x_stream, const void* y, long long ldy, const int* slots,
                               const float* weights, int top, const int* choice, int experts, const void* own, long long ld_own,
                               const void* shared, long long ld_shared, const void* gate, long long ld_gate, const void* w_out,
                               const void* mix, const void* w_in, const void* w_norm, float* x_out, void* h, long long rows, int n,
                               int cols, float eps, float scale, int dtype, cudaStream_t stream) {
  using namespace oslo;
  if (rows <= 0 || cols <= 0) return 0;
  if (rows > 0x7fffffffll || n < 1 || top < 0 || top > HYPER_MAX_TOP) return -1;
  HyperParams p{x, x_row, x_stream, y, ldy, slots, weights, choice, experts, own, ld_own, shared, ld_shared, gate, ld_gate,
                w_out, mix, w_in, w_norm, x_out, h, n, top, cols, eps, scale};
  const size_t te = dtype == OSLO_DT_FP32 ? 4 : 2;
  bool vec = cols % 4 == 0 && x_row % 4 == 0 && x_stream % 4 == 0 && ldy % 4 == 0 && ld_own % 4 == 0 && ld_shared % 4 == 0 &&
             aligned_to(x, 16) && aligned_to(x_out, 16);
  for (const void* t : {y, own, shared, w_norm, static_cast<const void*>(h)}) vec = vec && aligned_to(t, 4 * te);   // null is aligned
  OSLO_DISPATCH_T(dtype, { return vec ? hyper_dispatch<T, 4>(p, rows, stream) : hyper_dispatch<T, 1>(p, rows, stream); });
  return -2;
}
