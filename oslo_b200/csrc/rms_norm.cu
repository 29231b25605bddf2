// RMS norms with 32-bit arithmetic and the step that joins a sublayer to the residual stream.
//
//   rms_norm:      out = x / sqrt(mean(x^2) + eps) * (offset + w)        offset 1: the weight is stored around zero; w may be one number
//   gated_rms_norm: out = o / sqrt(mean(o^2 of a run of columns) + eps) * w * act(gate); the runs may first be divided by
//                  max(|z|, exp(-m)) + 1e-6, one z and m per run
//   branch_join:   x'  = x + mult * sum of the (possibly normed or scaled) results of parallel branches
//                  h_i = x' / sqrt(mean(x'^2) + eps) * w_i, i = 1, 2    the inputs of the next layer's branches, or a copy of x'; in a
//                  decode step also h_1 + conv(h_1), the convolution over the token and its predecessors (a state)
//   token_gate:    out = gelu_tanh(z) * the token's entries of a table
//   residual_join: z   = y * sigmoid(gate + gate_bias)
//                  x'  = x + z / sqrt(mean(z^2) + eps) * (1 + w_post)
//                  h   = x' / sqrt(mean(x'^2) + eps) * (1 + w_next)      the input of the next sublayer, 16-bit
// The residual stream x is 32-bit. y is either one row per token or the weighted sum of the `top` rows that a
// mixture-of-experts layer left in its slot buffer, so that the experts' combine step costs no pass of its own.
#include <algorithm>

#include "num.cuh"
#include "oslo_kernels.h"
#include "ptx.cuh"

namespace oslo {

// weights c.. of a norm, or (one) its only number
template <typename T, int VEC>
__device__ __forceinline__ void load_weight(const void* w, int one, int c, float (&v)[VEC]) {
  if (one) {
    const float g = Num<T>::to(*static_cast<const T*>(w));
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = g;
  } else {
    load_vec<T, VEC>(static_cast<const T*>(w) + c, v);
  }
}

// one warp per row
template <typename TX, typename T, int VEC>
__global__ void __launch_bounds__(256) rms_norm_warp_kernel(const TX* __restrict__ x, long long ldx, const T* __restrict__ w,
                                                            T* __restrict__ out, long long ldo, long long rows, int cols,
                                                            float eps, float offset, int one) {
  const long long row = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (row >= rows) return;
  const TX* xr = x + row * ldx;
  float ss = 0.f;
  for (int c = lane * VEC; c < cols; c += 32 * VEC) {
    float v[VEC];
    load_vec<TX, VEC>(xr + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss = fmaf(v[i], v[i], ss);
  }
  ss = warp_sum(ss);
  const float r = 1.0f / sqrtf(ss / cols + eps);
  for (int c = lane * VEC; c < cols; c += 32 * VEC) {
    float v[VEC], g[VEC];
    load_vec<TX, VEC>(xr + c, v);
    load_weight<T, VEC>(w, one, c, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = v[i] * r * (offset + g[i]);
    store_vec<T, VEC>(out + row * ldo + c, v);
  }
}

// one block per row
template <typename TX, typename T, int VEC>
__global__ void __launch_bounds__(256) rms_norm_block_kernel(const TX* __restrict__ x, long long ldx, const T* __restrict__ w,
                                                             T* __restrict__ out, long long ldo, int cols, float eps,
                                                             float offset, int one) {
  __shared__ float red[32];
  const TX* xr = x + blockIdx.x * ldx;
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < cols; c += blockDim.x * VEC) {
    float v[VEC];
    load_vec<TX, VEC>(xr + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss = fmaf(v[i], v[i], ss);
  }
  ss = block_sum(ss, red);
  const float r = 1.0f / sqrtf(ss / cols + eps);
  for (int c = threadIdx.x * VEC; c < cols; c += blockDim.x * VEC) {
    float v[VEC], g[VEC];
    load_vec<TX, VEC>(xr + c, v);
    load_weight<T, VEC>(w, one, c, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = v[i] * r * (offset + g[i]);
    store_vec<T, VEC>(out + blockIdx.x * ldo + c, v);
  }
}

template <typename TX, typename T, int VEC>
static void rms_norm_launch(const void* x, long long ldx, const void* w, void* out, long long ldo, long long rows, int cols,
                            float eps, float offset, int one, cudaStream_t st) {
  if (cols <= 512 && rows >= 64) {
    rms_norm_warp_kernel<TX, T, VEC><<<static_cast<unsigned>((rows + 7) / 8), 256, 0, st>>>(
        static_cast<const TX*>(x), ldx, static_cast<const T*>(w), static_cast<T*>(out), ldo, rows, cols, eps, offset, one);
  } else {
    const int threads = cols >= 256 * VEC ? 256 : (cols >= 128 * VEC ? 128 : 64);
    rms_norm_block_kernel<TX, T, VEC><<<static_cast<unsigned>(rows), threads, 0, st>>>(
        static_cast<const TX*>(x), ldx, static_cast<const T*>(w), static_cast<T*>(out), ldo, cols, eps, offset, one);
  }
}

struct JoinParams {
  const float* x;
  const void* y; long long ldy;
  const int* slots;            // [rows, top] rows of y, or nullptr: row * top + j
  const float* slot_weights;   // [rows, top], or nullptr: y has one row per token
  int top;
  const void* gate; long long ldg;
  const void* gate_bias;
  const void* w_post;
  const void* w_next;          // nullptr: no second norm
  float* x_out;
  void* h_out;
  int cols;
  float eps;
};

template <typename T, int VEC>
__global__ void __launch_bounds__(256) residual_join_kernel(const JoinParams p) {
  extern __shared__ float row_s[];
  __shared__ float red[32];
  const long long row = blockIdx.x;
  const T* gate = static_cast<const T*>(p.gate) + row * p.ldg;
  const T* gb = static_cast<const T*>(p.gate_bias);
  const T* y = static_cast<const T*>(p.y);
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < p.cols; c += blockDim.x * VEC) {
    float z[VEC], g[VEC], b[VEC];
    if (p.slot_weights == nullptr) {
      load_vec<T, VEC>(y + row * p.ldy + c, z);
    } else {
#pragma unroll
      for (int i = 0; i < VEC; ++i) z[i] = 0.f;
      for (int j = 0; j < p.top; ++j) {
        const long long s = p.slots ? p.slots[row * p.top + j] : row * p.top + j;
        const float wgt = p.slot_weights[row * p.top + j];
        float e[VEC];
        load_vec<T, VEC>(y + s * p.ldy + c, e);
#pragma unroll
        for (int i = 0; i < VEC; ++i) z[i] = fmaf(wgt, e[i], z[i]);
      }
    }
    load_vec<T, VEC>(gate + c, g);
    load_vec<T, VEC>(gb + c, b);
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      z[i] *= sigmoid_f(g[i] + b[i]);
      ss = fmaf(z[i], z[i], ss);
      row_s[c + i] = z[i];
    }
  }
  ss = block_sum(ss, red);
  const float r = 1.0f / sqrtf(ss / p.cols + p.eps);
  const T* wp = static_cast<const T*>(p.w_post);
  float sx = 0.f;
  for (int c = threadIdx.x * VEC; c < p.cols; c += blockDim.x * VEC) {   // every thread revisits its own elements
    float v[VEC], w[VEC];
    load_vec<float, VEC>(p.x + row * p.cols + c, v);
    load_vec<T, VEC>(wp + c, w);
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      v[i] += row_s[c + i] * r * (1.0f + w[i]);
      sx = fmaf(v[i], v[i], sx);
      row_s[c + i] = v[i];
    }
    store_vec<float, VEC>(p.x_out + row * p.cols + c, v);
  }
  if (p.w_next == nullptr) return;
  sx = block_sum(sx, red);
  const float rn = 1.0f / sqrtf(sx / p.cols + p.eps);
  const T* wn = static_cast<const T*>(p.w_next);
  for (int c = threadIdx.x * VEC; c < p.cols; c += blockDim.x * VEC) {
    float v[VEC], w[VEC];
    load_vec<T, VEC>(wn + c, w);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = row_s[c + i] * rn * (1.0f + w[i]);
    store_vec<T, VEC>(static_cast<T*>(p.h_out) + row * p.cols + c, v);
  }
}

struct BranchParams {
  const float* x;
  int n;
  const void* y[3]; long long ldy[3];
  const void* w[3];            // norm weight of the branch, or (normed 0) what its result is multiplied by, or nullptr
  int normed[3];
  const int* slots[3];         // [rows, top] rows of y that are summed, or nullptr: row * top + j
  int top[3];                  // 0: one row of y per row
  float factor[3];
  float mult, eps;
  const void *w1, *w2;         // nullptr: no such output
  int one1, one2;              // the weight is one number
  int copy;                    // h1 is x' in T
  float* x_out;
  void *h1, *h2;
  int cols;
  // one token per row: conv_out = h1 + sum_j conv_w[., j] * (the row's last taps - 1 inputs in prev, then h1); prev moves on
  const void* conv_w;          // [cols, taps], or nullptr
  float* prev;                 // [rows, taps - 1, cols], or nullptr (zeros)
  int taps;
  const uint8_t* keep; long long ld_keep;   // 0: the row's token counts as zeros; or nullptr
  void* conv_out;
};

template <typename T, int VEC>
__device__ __forceinline__ void load_branch(const BranchParams& p, int b, long long row, int c, float (&v)[VEC]) {
  const T* y = static_cast<const T*>(p.y[b]);
  const int top = p.top[b];
  if (top == 0) {
    load_vec<T, VEC>(y + row * p.ldy[b] + c, v);
    return;
  }
#pragma unroll
  for (int i = 0; i < VEC; ++i) v[i] = 0.f;
  const int* slots = p.slots[b];
#pragma unroll 4
  for (int j = 0; j < top; ++j) {
    const long long s = slots ? static_cast<long long>(slots[row * top + j]) : row * top + j;
    float e[VEC];
    load_vec<T, VEC>(y + s * p.ldy[b] + c, e);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] += e[i];
  }
}

// THREADS: at most; few rows get large blocks, so that a row's loads are on their way together
template <typename T, int VEC, int THREADS>
__global__ void __launch_bounds__(THREADS) branch_join_kernel(const BranchParams p) {
  extern __shared__ float row_s[];
  __shared__ float red[32];
  const long long row = blockIdx.x;
  float f[3];
#pragma unroll
  for (int b = 0; b < 3; ++b) {
    if (b >= p.n) break;
    f[b] = p.mult * p.factor[b];
    if (p.w[b] == nullptr || !p.normed[b]) continue;   // uniform over the block
    float ss = 0.f;
    for (int c = threadIdx.x * VEC; c < p.cols; c += blockDim.x * VEC) {
      float v[VEC];
      load_branch<T, VEC>(p, b, row, c, v);
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss = fmaf(v[i], v[i], ss);
    }
    ss = block_sum(ss, red);
    f[b] *= 1.0f / sqrtf(ss / p.cols + p.eps);
  }
  float sx = 0.f;
  for (int c = threadIdx.x * VEC; c < p.cols; c += blockDim.x * VEC) {
    float v[VEC];
    load_vec<float, VEC>(p.x + row * p.cols + c, v);
#pragma unroll
    for (int b = 0; b < 3; ++b) {
      if (b >= p.n) break;
      float y[VEC];
      load_branch<T, VEC>(p, b, row, c, y);
      if (p.w[b] != nullptr) {
        float w[VEC];
        load_vec<T, VEC>(static_cast<const T*>(p.w[b]) + c, w);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = fmaf(f[b] * y[i], w[i], v[i]);
      } else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = fmaf(f[b], y[i], v[i]);
      }
    }
    store_vec<float, VEC>(p.x_out + row * p.cols + c, v);
    if (p.copy) store_vec<T, VEC>(static_cast<T*>(p.h1) + row * p.cols + c, v);
    if (p.w1 == nullptr) continue;
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      sx = fmaf(v[i], v[i], sx);
      row_s[c + i] = v[i];
    }
  }
  if (p.w1 == nullptr) return;
  sx = block_sum(sx, red);
  const float rn = 1.0f / sqrtf(sx / p.cols + p.eps);
  const bool real = p.keep == nullptr || p.keep[row * p.ld_keep] != 0;
  for (int c = threadIdx.x * VEC; c < p.cols; c += blockDim.x * VEC) {   // every thread revisits its own elements
    float v[VEC], w[VEC];
    load_weight<T, VEC>(p.w1, p.one1, c, w);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = row_s[c + i] * rn * w[i];
    store_vec<T, VEC>(static_cast<T*>(p.h1) + row * p.cols + c, v);
    if (p.conv_w != nullptr) {
      float o[VEC];
      const T* cw = static_cast<const T*>(p.conv_w) + static_cast<long long>(c) * p.taps;
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        v[i] = real ? Num<T>::to(Num<T>::from(v[i])) : 0.f;              // what a prompt's convolution reads
        o[i] = v[i] * (1.0f + Num<T>::to(cw[i * p.taps + p.taps - 1]));
      }
      if (p.prev != nullptr) {
        float* state = p.prev + row * (p.taps - 1) * p.cols + c;
        float s[VEC];
        for (int j = 0; j < p.taps - 1; ++j) {
          load_vec<float, VEC>(state + static_cast<long long>(j) * p.cols, s);
#pragma unroll
          for (int i = 0; i < VEC; ++i) o[i] = fmaf(s[i], Num<T>::to(cw[i * p.taps + j]), o[i]);
          if (j > 0) store_vec<float, VEC>(state + static_cast<long long>(j - 1) * p.cols, s);
        }
        if (p.taps > 1) store_vec<float, VEC>(state + static_cast<long long>(p.taps - 2) * p.cols, v);
      }
      store_vec<T, VEC>(static_cast<T*>(p.conv_out) + row * p.cols + c, o);
    }
    if (p.w2 != nullptr) {
      load_weight<T, VEC>(p.w2, p.one2, c, w);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = row_s[c + i] * rn * w[i];
      store_vec<T, VEC>(static_cast<T*>(p.h2) + row * p.cols + c, v);
    }
  }
}

// out[r, c] = gelu_tanh(z[r, c]) * table[ids[r], first + c]; a token outside the table counts as one with zeros
template <typename T, int VEC>
__global__ void __launch_bounds__(256) token_gate_kernel(const T* __restrict__ z, long long ldz, const long long* __restrict__ ids,
                                                         long long id_step, const T* __restrict__ table, long long ldt, long long vocab, int first,
                                                         T* __restrict__ out, long long rows, int cols, int* err) {
  const int per_row = cols / VEC;
  const long long total = rows * per_row;
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < total;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long r = i / per_row;
    const int c = static_cast<int>(i - r * per_row) * VEC;
    const long long id = ids[r * id_step];
    float a[VEC], e[VEC];
    load_vec<T, VEC>(z + r * ldz + c, a);
    if (id >= 0 && id < vocab) {
      load_vec<T, VEC>(table + id * ldt + first + c, e);
    } else {
      OSLO_REPORT_BOUNDS(err);
#pragma unroll
      for (int k = 0; k < VEC; ++k) e[k] = 0.f;
    }
#pragma unroll
    for (int k = 0; k < VEC; ++k) {
      const float u = 0.7978845608028654f * (a[k] + 0.044715f * a[k] * a[k] * a[k]);
      a[k] = 0.5f * a[k] * (1.0f + tanhf(u)) * e[k];
    }
    store_vec<T, VEC>(out + r * cols + c, a);
  }
}

template <typename T, int VEC>
__device__ __forceinline__ void gate_run(const float* o, const T* w, const T* gate, T* out, int c, float r, int act) {
  float v[VEC], g[VEC], ww[VEC];
  load_vec<float, VEC>(o + c, v);
  load_vec<T, VEC>(w + c, ww);
  load_vec<T, VEC>(gate + c, g);
#pragma unroll
  for (int i = 0; i < VEC; ++i) v[i] = v[i] * r * ww[i] * (act ? silu_f(g[i]) : sigmoid_f(g[i]));
  store_vec<T, VEC>(out + c, v);
}

// LANES lanes of a warp per run of `group` columns, or (LANES 0) one block
template <typename T, int VEC, int LANES>
__global__ void __launch_bounds__(256) gated_rms_norm_kernel(const float* __restrict__ o, const T* __restrict__ w,
                                                             const T* __restrict__ gate, long long ldg, T* __restrict__ out,
                                                             const float* __restrict__ z, const float* __restrict__ m,
                                                             long long runs, int cols, int group, float eps, int act) {
  __shared__ float red[32];
  constexpr bool WARP = LANES > 0;
  constexpr int L = WARP ? LANES : 32;
  const bool real = !WARP || static_cast<long long>(blockIdx.x) * (blockDim.x / L) + threadIdx.x / L < runs;
  // lanes past the last run repeat it without storing, so that their warp stays whole
  const long long run = WARP ? (real ? static_cast<long long>(blockIdx.x) * (blockDim.x / L) + threadIdx.x / L : runs - 1) : blockIdx.x;
  const int per_row = cols / group;
  const long long row = run / per_row;
  const int c0 = static_cast<int>(run - row * per_row) * group;
  const int lane = WARP ? threadIdx.x % L : threadIdx.x, step = WARP ? L : blockDim.x;
  o += row * cols + c0;
  w += c0;
  gate += row * ldg + c0;
  out += row * cols + c0;
  float ss = 0.f;
  for (int c = lane * VEC; c < group; c += step * VEC) {
    float v[VEC];
    load_vec<float, VEC>(o + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss = fmaf(v[i], v[i], ss);
  }
  if (WARP) {
#pragma unroll
    for (int off = L / 2; off > 0; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
  } else {
    ss = block_sum(ss, red);
  }
  if (!real) return;
  const float inv = z ? 1.0f / (fmaxf(fabsf(z[run]), expf(-m[run])) + 1e-6f) : 1.0f;
  const float r = inv / sqrtf(inv * inv * (ss / group) + eps);
  for (int c = lane * VEC; c < group; c += step * VEC) gate_run<T, VEC>(o, w, gate, out, c, r, act);
}

struct SiluUnit {
  __device__ __forceinline__ float operator()(float g, float u) const { return silu_f(g) * u; }
};
struct ClampedUnit {
  float limit, alpha;
  __device__ __forceinline__ float operator()(float g, float u) const {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g * sigmoid_f(alpha * g) * (u + 1.0f);
  }
};

// y = unit(gate, up) on [rows, cols] slices with row strides
template <typename T, int VEC, typename Unit>
__global__ void __launch_bounds__(256) gated_unit_kernel(const T* __restrict__ gate, long long ldg, const T* __restrict__ up,
                                                         long long ldu, T* __restrict__ out, long long rows, int cols,
                                                         const Unit unit) {
  const long long per_row = cols / VEC;
  const long long total = rows * per_row;
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < total;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long r = i / per_row;
    const int c = static_cast<int>(i - r * per_row) * VEC;
    float a[VEC], b[VEC];
    load_vec<T, VEC>(gate + r * ldg + c, a);
    load_vec<T, VEC>(up + r * ldu + c, b);
#pragma unroll
    for (int k = 0; k < VEC; ++k) a[k] = unit(a[k], b[k]);
    store_vec<T, VEC>(out + r * cols + c, a);
  }
}

template <typename Unit>
static int gated_unit(const void* gate, long long ldg, const void* up, long long ldu, void* out, long long rows, int cols,
                      const Unit& unit, int dtype, cudaStream_t stream) {
  if (rows <= 0 || cols <= 0) return 0;
  const size_t te = dtype == OSLO_DT_FP32 ? 4 : 2;
  const bool vec = cols % 4 == 0 && ldg % 4 == 0 && ldu % 4 == 0 && aligned_to(gate, 4 * te) && aligned_to(up, 4 * te) &&
                   aligned_to(out, 4 * te);
  const long long work = rows * (vec ? cols / 4 : cols);
  const unsigned blocks = static_cast<unsigned>(std::min<long long>((work + 255) / 256, 148 * 16));
  OSLO_DISPATCH_T(dtype, {
    if (vec) gated_unit_kernel<T, 4, Unit><<<blocks, 256, 0, stream>>>(static_cast<const T*>(gate), ldg, static_cast<const T*>(up),
                                                                       ldu, static_cast<T*>(out), rows, cols, unit);
    else gated_unit_kernel<T, 1, Unit><<<blocks, 256, 0, stream>>>(static_cast<const T*>(gate), ldg, static_cast<const T*>(up), ldu,
                                                                   static_cast<T*>(out), rows, cols, unit);
  });
  return static_cast<int>(cudaGetLastError());
}

}  // namespace oslo

extern "C" int oslo_rms_norm(const void* x, long long ldx, int x_fp32, const void* w, int one, void* out, long long ldo,
                             long long rows, int cols, float eps, float offset, int dtype, cudaStream_t stream) {
  using namespace oslo;
  if (rows <= 0 || cols <= 0) return 0;
  if (rows > 0x7fffffffll) return -1;
  const size_t xe = x_fp32 ? 4 : (dtype == OSLO_DT_FP32 ? 4 : 2), te = dtype == OSLO_DT_FP32 ? 4 : 2;
  const bool vec = cols % 4 == 0 && ldx % 4 == 0 && ldo % 4 == 0 && aligned_to(x, 4 * xe) && (one || aligned_to(w, 4 * te)) &&
                   aligned_to(out, 4 * te);
  OSLO_DISPATCH_T(dtype, {
    if (x_fp32) {
      if (vec) rms_norm_launch<float, T, 4>(x, ldx, w, out, ldo, rows, cols, eps, offset, one, stream);
      else rms_norm_launch<float, T, 1>(x, ldx, w, out, ldo, rows, cols, eps, offset, one, stream);
    } else {
      if (vec) rms_norm_launch<T, T, 4>(x, ldx, w, out, ldo, rows, cols, eps, offset, one, stream);
      else rms_norm_launch<T, T, 1>(x, ldx, w, out, ldo, rows, cols, eps, offset, one, stream);
    }
  });
  return static_cast<int>(cudaGetLastError());
}

extern "C" int oslo_residual_join(const float* x, const void* y, long long ldy, const int* slots, const float* slot_weights,
                                  int top, const void* gate, long long ldg, const void* gate_bias, const void* w_post,
                                  const void* w_next, float* x_out, void* h_out, long long rows, int cols, float eps,
                                  int dtype, cudaStream_t stream) {
  using namespace oslo;
  if (rows <= 0 || cols <= 0) return 0;
  if (rows > 0x7fffffffll) return -1;
  JoinParams p{x, y, ldy, slots, slot_weights, top, gate, ldg, gate_bias, w_post, w_next, x_out, h_out, cols, eps};
  const size_t te = dtype == OSLO_DT_FP32 ? 4 : 2;
  const bool vec = cols % 4 == 0 && ldy % 4 == 0 && ldg % 4 == 0 && aligned_to(x, 16) && aligned_to(x_out, 16) &&
                   aligned_to(y, 4 * te) && aligned_to(gate, 4 * te) && aligned_to(gate_bias, 4 * te) &&
                   aligned_to(w_post, 4 * te) && (w_next == nullptr || (aligned_to(w_next, 4 * te) && aligned_to(h_out, 4 * te)));
  const size_t smem = static_cast<size_t>(cols) * sizeof(float);
  if (smem > 200 * 1024) return -3;
  const int threads = cols >= 1024 ? 256 : (cols >= 512 ? 128 : 64);
#define JOIN_GO(V)                                                                                                 \
  {                                                                                                                \
    if (smem > 48 * 1024) {                                                                                        \
      cudaError_t e = cudaFuncSetAttribute(residual_join_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                           static_cast<int>(smem));                                                \
      if (e != cudaSuccess) return static_cast<int>(e);                                                            \
    }                                                                                                              \
    residual_join_kernel<T, V><<<static_cast<unsigned>(rows), threads, smem, stream>>>(p);                         \
  }
  OSLO_DISPATCH_T(dtype, { if (vec) JOIN_GO(4) else JOIN_GO(1) });
#undef JOIN_GO
  return static_cast<int>(cudaGetLastError());
}

extern "C" int oslo_silu_mul(const void* gate, long long ldg, const void* up, long long ldu, void* out, long long rows,
                             int cols, int dtype, cudaStream_t stream) {
  return oslo::gated_unit(gate, ldg, up, ldu, out, rows, cols, oslo::SiluUnit{}, dtype, stream);
}

extern "C" int oslo_clamped_glu(const void* gate, long long ldg, const void* up, long long ldu, void* out, long long rows,
                                int cols, float limit, float alpha, int dtype, cudaStream_t stream) {
  return oslo::gated_unit(gate, ldg, up, ldu, out, rows, cols, oslo::ClampedUnit{limit, alpha}, dtype, stream);
}

extern "C" int oslo_branch_join(const OsloBranchJoin* a, long long rows, int cols, int dtype, cudaStream_t stream) {
  using namespace oslo;
  if (rows <= 0 || cols <= 0) return 0;
  if (rows > 0x7fffffffll || a->n < 1 || a->n > 3 || (a->copy && a->w1) || (a->conv_w && (!a->w1 || a->taps < 1))) return -1;
  const size_t te = dtype == OSLO_DT_FP32 ? 4 : 2;
  BranchParams p{};
  bool vec = cols % 4 == 0 && aligned_to(a->x, 16) && aligned_to(a->x_out, 16) && aligned_to(a->prev, 16);
  for (const void* t : {static_cast<const void*>(a->h1), static_cast<const void*>(a->h2), static_cast<const void*>(a->conv_out),
                        a->one1 ? nullptr : a->w1, a->one2 ? nullptr : a->w2}) vec = vec && aligned_to(t, 4 * te);   // null is aligned
  p.x = a->x; p.n = a->n;
  for (int i = 0; i < p.n; ++i) {
    p.y[i] = a->y[i]; p.ldy[i] = a->ldy[i]; p.w[i] = a->w[i]; p.normed[i] = a->normed[i]; p.slots[i] = a->slots[i]; p.top[i] = a->top[i];
    p.factor[i] = a->factor[i];
    vec = vec && p.ldy[i] % 4 == 0 && aligned_to(p.y[i], 4 * te) && aligned_to(p.w[i], 4 * te);
  }
  p.mult = a->mult; p.eps = a->eps; p.w1 = a->w1; p.w2 = a->w2; p.one1 = a->one1; p.one2 = a->one2; p.copy = a->copy;
  p.x_out = a->x_out; p.h1 = a->h1; p.h2 = a->h2; p.cols = cols;
  p.conv_w = a->conv_w; p.prev = a->prev; p.taps = a->taps; p.keep = a->keep; p.ld_keep = a->ld_keep; p.conv_out = a->conv_out;
  const size_t smem = a->w1 ? static_cast<size_t>(cols) * sizeof(float) : 0;
  if (smem > 200 * 1024) return -3;
  const int threads = cols >= 1024 ? 256 : (cols >= 512 ? 128 : 64);
  const bool few = rows <= 296 && cols > 1024;         // at most two blocks per SM
#define BRANCH_GO(V, N, THREADS)                                                                                 \
  {                                                                                                              \
    if (smem > 48 * 1024) {                                                                                      \
      cudaError_t e = cudaFuncSetAttribute(branch_join_kernel<T, V, N>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                           static_cast<int>(smem));                                              \
      if (e != cudaSuccess) return static_cast<int>(e);                                                          \
    }                                                                                                            \
    branch_join_kernel<T, V, N><<<static_cast<unsigned>(rows), THREADS, smem, stream>>>(p);                      \
  }
  OSLO_DISPATCH_T(dtype, {
    if (vec && few) BRANCH_GO(4, 1024, std::min(1024, (cols / 4 + 31) / 32 * 32))
    else if (vec) BRANCH_GO(4, 256, threads)
    else BRANCH_GO(1, 256, threads)
  });
#undef BRANCH_GO
  return static_cast<int>(cudaGetLastError());
}

extern "C" int oslo_token_gate(const void* z, long long ldz, const long long* ids, long long id_step, const void* table, long long ldt,
                               long long vocab, int first, void* out, long long rows, int cols, int dtype, int* err_word, cudaStream_t stream) {
  using namespace oslo;
  if (rows <= 0 || cols <= 0) return 0;
  if (first < 0 || first + cols > ldt) return -1;
  const size_t te = dtype == OSLO_DT_FP32 ? 4 : 2;
  const bool vec = cols % 4 == 0 && ldz % 4 == 0 && ldt % 4 == 0 && first % 4 == 0 && aligned_to(z, 4 * te) && aligned_to(table, 4 * te) &&
                   aligned_to(out, 4 * te);
  const long long total = rows * (vec ? cols / 4 : cols);
  const unsigned blocks = static_cast<unsigned>(std::min<long long>((total + 255) / 256, 148 * 16));
#define TG_GO(V) token_gate_kernel<T, V><<<blocks, 256, 0, stream>>>(static_cast<const T*>(z), ldz, ids, id_step, static_cast<const T*>(table), ldt, \
                                                                     vocab, first, static_cast<T*>(out), rows, cols, err_word)
  OSLO_DISPATCH_T(dtype, { if (vec) TG_GO(4); else TG_GO(1); });
#undef TG_GO
  return static_cast<int>(cudaGetLastError());
}

extern "C" int oslo_gated_rms_norm(const float* o, const void* w, const void* gate, long long ldg, void* out, const float* z,
                                   const float* m, long long rows, int cols, int group, float eps, int act, int dtype,
                                   cudaStream_t stream) {
  using namespace oslo;
  if (rows <= 0 || cols <= 0) return 0;
  if (group <= 0 || cols % group || (z == nullptr) != (m == nullptr)) return -1;
  const long long runs = rows * (cols / group);
  if (runs > 0x7fffffffll) return -1;
  const size_t te = dtype == OSLO_DT_FP32 ? 4 : 2;
  const bool vec = group % 4 == 0 && ldg % 4 == 0 && aligned_to(o, 16) && aligned_to(w, 4 * te) && aligned_to(gate, 4 * te) &&
                   aligned_to(out, 4 * te);
#define GATED_LAUNCH(V, L, BLOCKS)                                                                  \
  gated_rms_norm_kernel<T, V, L><<<static_cast<unsigned>(BLOCKS), 256, 0, stream>>>(                \
      o, static_cast<const T*>(w), static_cast<const T*>(gate), ldg, static_cast<T*>(out), z, m, runs, cols, group, eps, act)
#define GATED_GO(V)                                                         \
  if (group <= 8 * V) GATED_LAUNCH(V, 8, (runs + 31) / 32);                 \
  else if (group <= 16 * V) GATED_LAUNCH(V, 16, (runs + 15) / 16);          \
  else if (group <= 512) GATED_LAUNCH(V, 32, (runs + 7) / 8);               \
  else GATED_LAUNCH(V, 0, runs);
  OSLO_DISPATCH_T(dtype, { if (vec) { GATED_GO(4) } else { GATED_GO(1) } });
#undef GATED_LAUNCH
#undef GATED_GO
  return static_cast<int>(cudaGetLastError());
}
