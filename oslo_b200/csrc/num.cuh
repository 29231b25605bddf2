// Element conversions and small device helpers shared by the kernels that keep their arithmetic in 32-bit floats
// whatever the storage type is (rms_norm.cu, linear_recurrence.cu, latent_attention.cu, moe.cu). Those files are
// compiled without --use_fast_math: the same kernels serve float32 models.
#pragma once
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace oslo {

template <typename T> struct Num;
template <> struct Num<float> {
  static __device__ __forceinline__ float to(float v) { return v; }
  static __device__ __forceinline__ float from(float v) { return v; }
};
template <> struct Num<__nv_bfloat16> {
  static __device__ __forceinline__ float to(__nv_bfloat16 v) { return __bfloat162float(v); }
  static __device__ __forceinline__ __nv_bfloat16 from(float v) { return __float2bfloat16_rn(v); }
};
template <> struct Num<__half> {
  static __device__ __forceinline__ float to(__half v) { return __half2float(v); }
  static __device__ __forceinline__ __half from(float v) { return __float2half_rn(v); }
};

// VEC consecutive elements as floats; VEC * sizeof(T) bytes, aligned to that size (VEC a power of two)
template <typename T, int VEC> struct alignas(sizeof(T) * VEC) Pack { T e[VEC]; };
template <typename T, int VEC>
__device__ __forceinline__ void load_vec(const T* p, float (&v)[VEC]) {
  const Pack<T, VEC> k = *reinterpret_cast<const Pack<T, VEC>*>(p);
#pragma unroll
  for (int i = 0; i < VEC; ++i) v[i] = Num<T>::to(k.e[i]);
}
template <typename T, int VEC>
__device__ __forceinline__ void store_vec(T* p, const float (&v)[VEC]) {
  Pack<T, VEC> k;
#pragma unroll
  for (int i = 0; i < VEC; ++i) k.e[i] = Num<T>::from(v[i]);
  *reinterpret_cast<Pack<T, VEC>*>(p) = k;
}

__device__ __forceinline__ float sigmoid_f(float z) { return __fdividef(1.0f, 1.0f + expf(-z)); }   // 2 ulp; 0 when expf overflows
__device__ __forceinline__ float silu_f(float z) { return z * sigmoid_f(z); }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int off = 16; off > 0; off >>= 1) v += __shfl_xor_sync(0xffffffffu, v, off);
  return v;
}
// sum over the block; `red` holds 32 floats of shared memory and may be reused after the call's second barrier
__device__ __forceinline__ float block_sum(float v, float* red) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = lane < warps ? red[lane] : 0.f;
  return warp_sum(t);
}

// dot product of a row of K elements with a float row in shared memory, strided over a warp's lanes
template <typename T, int VEC>
__device__ __forceinline__ float warp_dot(const T* __restrict__ w, const float* __restrict__ x, int K, int lane) {
  float acc = 0.f;
  for (int k = lane * VEC; k < K; k += 32 * VEC) {
    float v[VEC];
    load_vec<T, VEC>(w + k, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) acc = fmaf(v[i], x[k + i], acc);
  }
  return warp_sum(acc);
}

#define OSLO_DISPATCH_T(code, ...)                                        \
  switch (code) {                                                         \
    case OSLO_DT_BF16: { using T = __nv_bfloat16; __VA_ARGS__; break; }   \
    case OSLO_DT_FP16: { using T = __half; __VA_ARGS__; break; }          \
    case OSLO_DT_FP32: { using T = float; __VA_ARGS__; break; }           \
    default: return -2;                                                   \
  }

inline bool aligned_to(const void* p, size_t bytes) { return (reinterpret_cast<uintptr_t>(p) & (bytes - 1)) == 0; }

}  // namespace oslo
