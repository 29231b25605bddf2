// Token shift, causal convolution per channel and selective scan (Mamba form), arithmetic and states in 32-bit floats.
//
//   token shift:  out_i = h_t + (h_{t-1} - h_t) * mu_i           h_{-1}: the state (zero for a new sequence)
//   convolution:  y_t = bias + sum_j w_j x_{t - taps + 1 + j}, then silu(y_t), or y_t + x_t, or as it is
//   scan:         s_t = softplus(dt_t + dt_bias),  S[n] <- exp(s_t A[n]) S[n] + s_t x_t B_t[n],  A = -exp(a_log)
//                 out_t = (sum_n S[n] C_t[n] + d x_t) * silu(z_t)
//
// Scan over a prompt (selective_scan_kernel): G lanes share a channel, each keeps NS of its states in registers (more lanes than
// needed when there are few channels). A stage of
// tokens is fetched one stage ahead with cp.async; step sizes and s_t x_t are computed once per (token, channel), B and C are
// broadcast from shared memory, the outputs pass through shared memory to the gated, coalesced store. One exponential per
// state and token bounds it (16 per cycle and SM). When the channels do not fill the GPU the prompt is cut into chunks:
// local states of all chunks but the last from zero, a scan over the chunks (a chunk's decay is exp(A * its summed steps)), then
// every chunk again from its true initial state.
// Decode (scan_step_kernel): the step's projection, the state update and the gate in one launch.
// A token whose `keep` entry is 0 (padding, on the left) counts as zero input and leaves the state as it is.
#include <algorithm>

#include "num.cuh"
#include "oslo_kernels.h"

namespace oslo {

// ------------------------------------------------------------------ token shift
constexpr int TS_RUN = 16;   // tokens per thread

struct ShiftParams {
  const void* h; long long ldh;
  const void* mu;                            // [P, width]
  const uint8_t* keep; long long ld_keep;    // [B, S] or nullptr
  float* prev;                               // [B, width] or nullptr
  void* out;                                 // [P, B * S, width]
  long long rows;                            // B * S
  int S, width;
};

template <typename T, int VEC, int P>
__global__ void __launch_bounds__(128) token_shift_kernel(const ShiftParams p) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  if (c >= p.width) return;
  const int b = blockIdx.z, t0 = blockIdx.y * TS_RUN, t1 = min(p.S, t0 + TS_RUN);
  const T* h = static_cast<const T*>(p.h) + static_cast<long long>(b) * p.S * p.ldh + c;
  auto row = [&](int t, float (&v)[VEC]) {
    load_vec<T, VEC>(h + t * p.ldh, v);
    if (p.keep && !p.keep[b * p.ld_keep + t]) {
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = 0.f;
    }
  };
  float mu[P][VEC], before[VEC];
#pragma unroll
  for (int j = 0; j < P; ++j) load_vec<T, VEC>(static_cast<const T*>(p.mu) + static_cast<long long>(j) * p.width + c, mu[j]);
  float* prev = p.prev ? p.prev + static_cast<long long>(b) * p.width + c : nullptr;
  if (t0 > 0) {
    row(t0 - 1, before);
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) before[i] = prev ? prev[i] : 0.f;
  }
  for (int t = t0; t < t1; ++t) {
    float now[VEC], y[VEC];
    row(t, now);
    T* out = static_cast<T*>(p.out) + (static_cast<long long>(b) * p.S + t) * p.width + c;
#pragma unroll
    for (int j = 0; j < P; ++j) {
#pragma unroll
      for (int i = 0; i < VEC; ++i) y[i] = fmaf(before[i] - now[i], mu[j][i], now[i]);
      store_vec<T, VEC>(out + j * p.rows * p.width, y);
    }
#pragma unroll
    for (int i = 0; i < VEC; ++i) before[i] = now[i];
  }
  if (t0 == 0 && prev) {                     // only this thread reads or writes these entries of the state
    row(p.S - 1, before);
#pragma unroll
    for (int i = 0; i < VEC; ++i) prev[i] = before[i];
  }
}

// ------------------------------------------------------------------ causal convolution
struct ConvParams {
  const void* x; long long ldx;
  const void *w, *bias;                      // [C, taps], [C] or nullptr
  const uint8_t* keep; long long ld_keep;
  float* prev;                               // [B, taps - 1, C] or nullptr
  void* out;                                 // [B * S, C]
  int S, C, taps, run;                       // run: tokens per thread, at least taps
  int silu, residual;
};

// TAPS 0: any number of taps, the window is read again for every token
template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(128) causal_conv_kernel(const ConvParams p) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  if (c >= p.C) return;
  const int taps = TAPS ? TAPS : p.taps;
  const int b = blockIdx.z, t0 = blockIdx.y * p.run, t1 = min(p.S, t0 + p.run);
  const T* x = static_cast<const T*>(p.x) + static_cast<long long>(b) * p.S * p.ldx + c;
  const T* w = static_cast<const T*>(p.w) + static_cast<long long>(c) * taps;
  float* prev = p.prev ? p.prev + static_cast<long long>(b) * (taps - 1) * p.C + c : nullptr;
  auto input = [&](int t, float (&v)[VEC]) {
    if (t >= 0) {
      load_vec<T, VEC>(x + t * p.ldx, v);
      if (p.keep && !p.keep[b * p.ld_keep + t]) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = 0.f;
      }
    } else {
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = prev ? prev[static_cast<long long>(t + taps - 1) * p.C + i] : 0.f;
    }
  };
  float bias[VEC];
#pragma unroll
  for (int i = 0; i < VEC; ++i) bias[i] = 0.f;
  if (p.bias != nullptr) load_vec<T, VEC>(static_cast<const T*>(p.bias) + c, bias);
  T* out = static_cast<T*>(p.out) + static_cast<long long>(b) * p.S * p.C + c;
  auto finish = [&](float y, float x) {
    if (p.residual) return y + x;
    if (!p.silu) return y;
    return sizeof(T) == 4 ? silu_f(y) : y * __fdividef(1.0f, 1.0f + __expf(-y));
  };
  if constexpr (TAPS > 0) {
    float wr[TAPS][VEC], win[TAPS][VEC];
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
      for (int i = 0; i < VEC; ++i) wr[j][i] = Num<T>::to(w[i * TAPS + j]);
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) input(t0 - TAPS + 1 + j, win[j + 1]);
    constexpr int AHEAD = 4;                 // tokens whose inputs are on their way
    for (int tb = t0; tb < t1; tb += AHEAD) {
      float now[AHEAD][VEC];
#pragma unroll
      for (int a = 0; a < AHEAD; ++a)
        if (tb + a < t1) input(tb + a, now[a]);
#pragma unroll
      for (int a = 0; a < AHEAD; ++a) {
        if (tb + a >= t1) break;
        float y[VEC];
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
          for (int i = 0; i < VEC; ++i) win[j][i] = win[j + 1][i];
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          win[TAPS - 1][i] = now[a][i];
          y[i] = bias[i];
#pragma unroll
          for (int j = 0; j < TAPS; ++j) y[i] = fmaf(wr[j][i], win[j][i], y[i]);
          y[i] = finish(y[i], now[a][i]);
        }
        store_vec<T, VEC>(out + static_cast<long long>(tb + a) * p.C, y);
      }
    }
  } else {
    for (int t = t0; t < t1; ++t) {
      float y[VEC], v[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) y[i] = bias[i];
      for (int j = 0; j < taps; ++j) {                 // the last one leaves the token's own input in v
        input(t - taps + 1 + j, v);
#pragma unroll
        for (int i = 0; i < VEC; ++i) y[i] = fmaf(Num<T>::to(w[i * taps + j]), v[i], y[i]);
      }
#pragma unroll
      for (int i = 0; i < VEC; ++i) y[i] = finish(y[i], v[i]);
      store_vec<T, VEC>(out + static_cast<long long>(t) * p.C, y);
    }
  }
  if (t0 == 0 && prev) {                     // the first run alone looks at the state (run >= taps); entries move towards the front
    for (int j = 0; j < taps - 1; ++j) {
      float v[VEC];
      input(p.S - taps + 1 + j, v);
#pragma unroll
      for (int i = 0; i < VEC; ++i) prev[static_cast<long long>(j) * p.C + i] = v[i];
    }
  }
}

// ------------------------------------------------------------------ selective scan, prompts
constexpr int SC_TB = 16;        // tokens staged at a time
constexpr int SC_THREADS = 128;
constexpr float SC_LOG2E = 1.4426950408889634f;

// 32-bit models get the accurate functions
template <typename T> __device__ __forceinline__ float softplus_t(float z) {
  if (sizeof(T) == 4) return z > 20.f ? z : log1pf(expf(z));
  // max(z, 0) + log(1 + e), e = exp(-|z|): log(1 + e) = 2 atanh(r), r = e / (2 + e) <= 1/3, by the series of atanh (the first term
  // left out is below 1e-8 of the sum); small e keep their relative precision
  const float e = __expf(-fabsf(z)), r = __fdividef(e, 2.f + e), q = r * r;
  float s = fmaf(q, 1.f / 15.f, 1.f / 13.f);
  s = fmaf(q, s, 1.f / 11.f);
  s = fmaf(q, s, 1.f / 9.f);
  s = fmaf(q, s, 1.f / 7.f);
  s = fmaf(q, s, 1.f / 5.f);
  s = fmaf(q, s, 1.f / 3.f);
  s = fmaf(q, s, 1.f);
  return fmaf(2.f * r, s, fmaxf(z, 0.f));
}
// exp(a): 16-bit models pass a * log2(e)
template <typename T> __device__ __forceinline__ float decay_t(float a) {
  if (sizeof(T) == 4) return expf(a);
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(a));
  return r;
}
template <typename T> __device__ __forceinline__ float decay_rate(float a_log) {
  return sizeof(T) == 4 ? -expf(a_log) : -__expf(a_log) * SC_LOG2E;
}

struct ScanParams {
  const void* x; long long ldx;
  const float* dt; long long lddt;           // step logits without the bias
  const void *dt_bias, *a_log, *d;           // [C], [C, N], [C]
  const void *b, *c; long long ldb, ldc;     // rows of N
  const void* z; long long ldz;
  const uint8_t* keep; long long ld_keep;
  void* out;                                 // [B * S, C]
  int B, S, C, N, NP;                        // NP: N rounded up to the states that a channel's lanes hold
  int chunk, nchunks;                        // tokens per chunk; chunks of this launch per batch row
  const float* s_in;                         // initial states, or nullptr (zero)
  float* s_out;                              // final states, or nullptr
  float* s_end;                              // last chunk only: final states [B, C, N], or nullptr
  long long s_batch, s_chunk;                // element strides of s_in / s_out over batch rows and chunks
  float* steps;                              // STATE_ONLY: sum of the chunk's steps [B, nchunks, C]
  int vec16;                                 // rows of dt, x and z start at 16-byte boundaries, C is a multiple of 8
  int bc16;                                  // rows of b and c start at 16-byte boundaries, N is a multiple of 8
};

template <typename T, int NS, int G, bool STATE_ONLY>
__global__ void __launch_bounds__(SC_THREADS) selective_scan_kernel(const ScanParams p) {
  constexpr int CH = SC_THREADS / G, NP = NS * G;
  extern __shared__ float4 sc_smem[];
  float* bs = reinterpret_cast<float*>(sc_smem);         // [SC_TB][NP]
  float* cs = bs + SC_TB * NP;                           // [SC_TB][NP], not STATE_ONLY
  float* step_s = cs + (STATE_ONLY ? 0 : SC_TB * NP);    // [SC_TB][CH]
  float* sx_s = step_s + SC_TB * CH;                     // [SC_TB][CH]: step * x
  float* y_s = sx_s + SC_TB * CH;                        // [SC_TB][CH], not STATE_ONLY
  float* draw = y_s + (STATE_ONLY ? 0 : SC_TB * CH);     // [2][SC_TB][CH] raw step logits
  T* xraw = reinterpret_cast<T*>(draw + 2 * SC_TB * CH); // [2][SC_TB][CH]
  T* braw = xraw + 2 * SC_TB * CH;                       // [2][SC_TB][NP8]
  constexpr int NP8 = (NP + 7) / 8 * 8;
  T* craw = braw + 2 * SC_TB * NP8;                      // [2][SC_TB][NP8], not STATE_ONLY
  T* zraw = craw + (STATE_ONLY ? 0 : 2 * SC_TB * NP8);   // [2][SC_TB][CH], not STATE_ONLY
  const int tid = threadIdx.x, g = tid % G, ch = tid / G;
  const int b = blockIdx.y / p.nchunks, ck = blockIdx.y % p.nchunks;
  const int c0 = blockIdx.x * CH, nc = min(CH, p.C - c0), my_c = c0 + ch;
  const int t_begin = ck * p.chunk, t_end = min(p.S, t_begin + p.chunk);
  const long long row0 = static_cast<long long>(b) * p.S;
  const T* x = static_cast<const T*>(p.x) + row0 * p.ldx + c0;
  const T* z = static_cast<const T*>(p.z) + row0 * p.ldz + c0;
  const float* dt = p.dt + row0 * p.lddt + c0;
  const T* bt = static_cast<const T*>(p.b) + row0 * p.ldb;
  const T* ct = static_cast<const T*>(p.c) + row0 * p.ldc;

  float s[NS], a[NS];
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const int n = g * NS + i;
    const bool real = ch < nc && n < p.N;
    a[i] = real ? decay_rate<T>(Num<T>::to(static_cast<const T*>(p.a_log)[static_cast<long long>(my_c) * p.N + n])) : 0.f;
    s[i] = real && !STATE_ONLY && p.s_in ? p.s_in[b * p.s_batch + ck * p.s_chunk + static_cast<long long>(my_c) * p.N + n] : 0.f;
  }
  auto fetch = [&](int t0, int buf) {
    const int n = min(SC_TB, t_end - t0);
    float* dd = draw + buf * SC_TB * CH;
    T* xd = xraw + buf * SC_TB * CH;
    T* zd = zraw + buf * SC_TB * CH;
    if (p.vec16) {
      constexpr int V = 16 / sizeof(T);
      for (int e = tid; e < n * (CH / 4); e += SC_THREADS) {
        const int t = e / (CH / 4), c = e % (CH / 4) * 4;
        if (c < nc) {
          const uint32_t d32 = static_cast<uint32_t>(__cvta_generic_to_shared(dd + t * CH + c));
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d32), "l"(dt + (t0 + t) * p.lddt + c) : "memory");
        }
      }
      for (int e = tid; e < n * (CH / V); e += SC_THREADS) {
        const int t = e / (CH / V), c = e % (CH / V) * V;
        if (c < nc) {
          const uint32_t x32 = static_cast<uint32_t>(__cvta_generic_to_shared(xd + t * CH + c));
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(x32), "l"(x + (t0 + t) * p.ldx + c) : "memory");
          if (!STATE_ONLY) {
            const uint32_t z32 = static_cast<uint32_t>(__cvta_generic_to_shared(zd + t * CH + c));
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(z32), "l"(z + (t0 + t) * p.ldz + c) : "memory");
          }
        }
      }
    } else {
      for (int e = tid; e < n * CH; e += SC_THREADS) {
        const int t = e / CH, c = e % CH;
        if (c < nc) {
          dd[e] = dt[(t0 + t) * p.lddt + c];
          xd[e] = x[(t0 + t) * p.ldx + c];
          if (!STATE_ONLY) zd[e] = z[(t0 + t) * p.ldz + c];
        }
      }
    }
    T* bd = braw + buf * SC_TB * NP8;
    T* cd = craw + buf * SC_TB * NP8;
    if (p.bc16) {
      constexpr int V = 16 / sizeof(T);
      for (int e = tid; e < n * (NP8 / V); e += SC_THREADS) {
        const int t = e / (NP8 / V), i = e % (NP8 / V) * V;
        if (i < p.N) {
          const uint32_t b32 = static_cast<uint32_t>(__cvta_generic_to_shared(bd + t * NP8 + i));
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(b32), "l"(bt + (t0 + t) * p.ldb + i) : "memory");
          if (!STATE_ONLY) {
            const uint32_t c32 = static_cast<uint32_t>(__cvta_generic_to_shared(cd + t * NP8 + i));
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(c32), "l"(ct + (t0 + t) * p.ldc + i) : "memory");
          }
        }
      }
    } else {
      for (int e = tid; e < n * NP8; e += SC_THREADS) {
        const int t = e / NP8, i = e % NP8;
        if (i < p.N) {
          bd[e] = bt[(t0 + t) * p.ldb + i];
          if (!STATE_ONLY) cd[e] = ct[(t0 + t) * p.ldc + i];
        }
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  float total = 0.f;
  if (t_begin < t_end) fetch(t_begin, 0);
  for (int t0 = t_begin, it = 0; t0 < t_end; t0 += SC_TB, ++it) {
    const int n = min(SC_TB, t_end - t0), buf = it & 1;
    if (t0 + SC_TB < t_end) {                            // every thread read the other stage before the last barrier
      fetch(t0 + SC_TB, buf ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    for (int e = tid; e < n * NP; e += SC_THREADS) {
      const int t = e / NP, i = e % NP;
      bs[e] = i < p.N ? Num<T>::to(braw[(buf * SC_TB + t) * NP8 + i]) : 0.f;
      if (!STATE_ONLY) cs[e] = i < p.N ? Num<T>::to(craw[(buf * SC_TB + t) * NP8 + i]) : 0.f;
    }
    {
      const int c = tid % CH;
      const float bias = c < nc ? Num<T>::to(static_cast<const T*>(p.dt_bias)[c0 + c]) : 0.f;
      for (int t = tid / CH; t < n; t += G) {
        const bool on = c < nc && (p.keep == nullptr || p.keep[b * p.ld_keep + t0 + t]);
        const float st = on ? softplus_t<T>(draw[(buf * SC_TB + t) * CH + c] + bias) : 0.f;
        step_s[t * CH + c] = st;
        sx_s[t * CH + c] = on ? st * Num<T>::to(xraw[(buf * SC_TB + t) * CH + c]) : 0.f;
      }
    }
    __syncthreads();
#pragma unroll 2
    for (int t = 0; t < n; ++t) {
      const float st = step_s[t * CH + ch], sx = sx_s[t * CH + ch];
      if (STATE_ONLY) total += st;
      float y0 = 0.f, y1 = 0.f;
#pragma unroll
      for (int i = 0; i < NS; i += 4) {
        const float4 b4 = *reinterpret_cast<const float4*>(bs + t * NP + g * NS + i);
        s[i] = fmaf(decay_t<T>(st * a[i]), s[i], sx * b4.x);
        s[i + 1] = fmaf(decay_t<T>(st * a[i + 1]), s[i + 1], sx * b4.y);
        s[i + 2] = fmaf(decay_t<T>(st * a[i + 2]), s[i + 2], sx * b4.z);
        s[i + 3] = fmaf(decay_t<T>(st * a[i + 3]), s[i + 3], sx * b4.w);
        if (!STATE_ONLY) {
          const float4 c4 = *reinterpret_cast<const float4*>(cs + t * NP + g * NS + i);
          y0 = fmaf(s[i], c4.x, y0);
          y1 = fmaf(s[i + 1], c4.y, y1);
          y0 = fmaf(s[i + 2], c4.z, y0);
          y1 = fmaf(s[i + 3], c4.w, y1);
        }
      }
      if (!STATE_ONLY) {
        float y = y0 + y1;
#pragma unroll
        for (int off = G / 2; off > 0; off >>= 1) y += __shfl_xor_sync(0xffffffffu, y, off);
        if (g == 0) y_s[t * CH + ch] = y;
      }
    }
    __syncthreads();
    if (!STATE_ONLY) {                                   // this stage's raw x and z are fetched over after the next barrier only
      const int c = tid % CH;
      if (c < nc) {
        const float d = Num<T>::to(static_cast<const T*>(p.d)[c0 + c]);
        T* out = static_cast<T*>(p.out) + (row0 + t0) * p.C + c0 + c;
        for (int t = tid / CH; t < n; t += G) {
          const float y = fmaf(d, Num<T>::to(xraw[(buf * SC_TB + t) * CH + c]), y_s[t * CH + c]);
          const float zz = Num<T>::to(zraw[(buf * SC_TB + t) * CH + c]);
          out[static_cast<long long>(t) * p.C] = Num<T>::from(y * (sizeof(T) == 4 ? silu_f(zz) : zz * __fdividef(1.0f, 1.0f + __expf(-zz))));
        }
      }
      __syncthreads();
    }
  }
  if (ch < nc) {
#pragma unroll
    for (int i = 0; i < NS; ++i) {
      const int n = g * NS + i;
      if (n < p.N) {
        const long long at = static_cast<long long>(my_c) * p.N + n;
        if (p.s_out) p.s_out[b * p.s_batch + ck * p.s_chunk + at] = s[i];
        if (p.s_end && ck == p.nchunks - 1) p.s_end[static_cast<long long>(b) * p.C * p.N + at] = s[i];
      }
    }
    if (STATE_ONLY && g == 0) p.steps[(static_cast<long long>(b) * p.nchunks + ck) * p.C + my_c] = total;
  }
}

// ws[b, k] (k < nchunks - 1) holds the local final state of chunk k; replace every ws[b, k] by the state at the chunk's start
template <typename T>
__global__ void __launch_bounds__(256) scan_chunks_kernel(float* __restrict__ ws, const float* __restrict__ steps,
                                                          const float* __restrict__ s_in, const T* __restrict__ a_log, int nchunks,
                                                          int C, int N) {
  const long long per = static_cast<long long>(C) * N;
  const long long e = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  const int b = blockIdx.y;
  if (e >= per) return;
  const long long ch = e / N;
  const float a = -expf(Num<T>::to(a_log[e]));
  float s = s_in ? s_in[b * per + e] : 0.f;
#pragma unroll 4
  for (int k = 0; k < nchunks; ++k) {
    const long long o = (static_cast<long long>(b) * nchunks + k) * per + e;
    const bool more = k + 1 < nchunks;
    const float local = more ? ws[o] : 0.f;
    const float d = more ? expf(a * steps[(static_cast<long long>(b) * (nchunks - 1) + k) * C + ch]) : 0.f;
    ws[o] = s;
    s = fmaf(d, s, local);
  }
}

// ------------------------------------------------------------------ selective scan, one token per row
constexpr int ST_CH = 32, ST_ROWS = 8;   // channels and rows of a block
constexpr int ST_PARTS = 4;              // MMA: warps that share the step projection of 16 channels

// D[channel][row] += W[channel][k] dt[row][k] for 16 channels, 8 rows and 16 k
__device__ __forceinline__ void st_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1, __nv_bfloat16) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void st_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1, __half) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void st_mma(float (&)[4], const uint32_t (&)[4], uint32_t, uint32_t, float) {}

struct ScanStepParams {
  const void* x; long long ldx;
  const void* dt; long long lddt;            // [B, rank]
  const void* w_dt; int rank;                // [C, rank]
  const void *dt_bias, *a_log, *d;
  const void *b, *c; long long ldb, ldc;
  const void* z; long long ldz;
  const uint8_t* keep; long long ld_keep;
  float* state;                              // [B, C, N]
  void* out;                                 // [B, C]
  int B, C, N;
};

// thread = (row, channel). MMA (16-bit types, rank a multiple of 16, even strides): the step projection on tensor cores
template <typename T, int VEC, int SVEC, bool MMA>
__global__ void __launch_bounds__(256) scan_step_kernel(const ScanStepParams p) {
  extern __shared__ float4 st_smem[];
  __shared__ float part[MMA ? ST_PARTS : 1][MMA ? ST_CH : 1][MMA ? ST_ROWS + 1 : 1];
  const int ldd = (p.rank + 3) / 4 * 4, ldw = ldd + 4;   // reads of four elements by 32 rows without conflicts
  float* bs = reinterpret_cast<float*>(st_smem);         // [ST_ROWS][N]
  float* cs = bs + ST_ROWS * p.N;                        // [ST_ROWS][N]
  float* dts = cs + ST_ROWS * p.N;                       // [ST_ROWS][ldd], not MMA
  T* ws = reinterpret_cast<T*>(dts + ST_ROWS * ldd);     // [ST_CH][ldw], not MMA
  const int tid = threadIdx.x, lane = tid & 31, r = tid >> 5;
  const int c0 = blockIdx.x * ST_CH, b0 = blockIdx.y * ST_ROWS, nb = min(ST_ROWS, p.B - b0), nc = min(ST_CH, p.C - c0);
  const int c = c0 + lane, b = b0 + r;
  const bool mine = r < nb && c < p.C;
  constexpr int AHEAD = 16 / SVEC;                       // states that are on their way while the step is computed
  float* s = p.state + (static_cast<long long>(b) * p.C + c) * p.N;
  float ahead[AHEAD][SVEC];
#pragma unroll
  for (int a = 0; a < AHEAD; ++a)
    if (mine && a * SVEC < p.N) load_vec<float, SVEC>(s + a * SVEC, ahead[a]);
  if constexpr (MMA) {
    const int j = (r & 1) * 16 + lane / 4, k2 = lane % 4 * 2;             // channels j and j + 8 of the fragments; row lane / 4
    const T* w0 = static_cast<const T*>(p.w_dt) + static_cast<long long>(c0 + j) * p.rank + k2;
    const T* w1 = w0 + 8ll * p.rank;
    const T* d = static_cast<const T*>(p.dt) + (b0 + lane / 4) * p.lddt + k2;
    const bool on0 = j < nc, on1 = j + 8 < nc, row = lane / 4 < nb;
    float z[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 2
    for (int k = r / 2 * 16; k < p.rank; k += 16 * ST_PARTS) {
      auto pair = [&](bool ok, const T* at) { return ok ? *reinterpret_cast<const uint32_t*>(at + k) : 0u; };
      const uint32_t a[4] = {pair(on0, w0), pair(on1, w1), pair(on0, w0 + 8), pair(on1, w1 + 8)};
      st_mma(z, a, pair(row, d), pair(row, d + 8), T());
    }
    part[r / 2][j][k2] = z[0];
    part[r / 2][j][k2 + 1] = z[1];
    part[r / 2][j + 8][k2] = z[2];
    part[r / 2][j + 8][k2 + 1] = z[3];
  } else {
    for (int j = tid / 8; j < nc; j += 32) {             // eight threads per row of the step projection
      const T* w = static_cast<const T*>(p.w_dt) + static_cast<long long>(c0 + j) * p.rank;
#pragma unroll 4
      for (int k = tid % 8 * VEC; k < p.rank; k += 8 * VEC)
        *reinterpret_cast<Pack<T, VEC>*>(ws + j * ldw + k) = *reinterpret_cast<const Pack<T, VEC>*>(w + k);
    }
  }
  if (r < nb) {                                          // a warp per row
    if (!MMA)
      for (int k = lane; k < ldd; k += 32) dts[r * ldd + k] = k < p.rank ? Num<T>::to(static_cast<const T*>(p.dt)[b * p.lddt + k]) : 0.f;
    for (int k = lane; k < p.N; k += 32) {
      bs[r * p.N + k] = Num<T>::to(static_cast<const T*>(p.b)[b * p.ldb + k]);
      cs[r * p.N + k] = Num<T>::to(static_cast<const T*>(p.c)[b * p.ldc + k]);
    }
  }
  __syncthreads();
  if (!mine) return;
  float st = 0.f;
  if (p.keep == nullptr || p.keep[b * p.ld_keep]) {
    float z0 = 0.f, z1 = 0.f;
    int k = 0;
    if constexpr (MMA) {
#pragma unroll
      for (int u = 0; u < ST_PARTS; ++u) z0 += part[u][lane][r];
      k = p.rank;
    } else if (VEC >= 4) {
#pragma unroll 4
      for (; k + 4 <= p.rank; k += 4) {
        float w[4];
        load_vec<T, 4>(ws + lane * ldw + k, w);
        const float4 d4 = *reinterpret_cast<const float4*>(dts + r * ldd + k);
        z0 = fmaf(w[0], d4.x, fmaf(w[1], d4.y, z0));
        z1 = fmaf(w[2], d4.z, fmaf(w[3], d4.w, z1));
      }
    }
    for (; k < p.rank; ++k) z0 = fmaf(Num<T>::to(ws[lane * ldw + k]), dts[r * ldd + k], z0);
    st = softplus_t<T>(z0 + z1 + Num<T>::to(static_cast<const T*>(p.dt_bias)[c]));
  }
  const float x = Num<T>::to(static_cast<const T*>(p.x)[b * p.ldx + c]), sx = st * x;
  const T* al = static_cast<const T*>(p.a_log) + static_cast<long long>(c) * p.N;
  float y = 0.f;
  auto update = [&](int n, float (&sv)[SVEC]) {
    float av[SVEC], bv[SVEC], cv[SVEC];
    load_vec<T, SVEC>(al + n, av);
    load_vec<float, SVEC>(bs + r * p.N + n, bv);
    load_vec<float, SVEC>(cs + r * p.N + n, cv);
#pragma unroll
    for (int i = 0; i < SVEC; ++i) {
      sv[i] = fmaf(decay_t<T>(st * decay_rate<T>(av[i])), sv[i], sx * bv[i]);
      y = fmaf(sv[i], cv[i], y);
    }
    store_vec<float, SVEC>(s + n, sv);
  };
#pragma unroll
  for (int a = 0; a < AHEAD; ++a)
    if (a * SVEC < p.N) update(a * SVEC, ahead[a]);
#pragma unroll 2
  for (int n = 16; n < p.N; n += SVEC) {
    float sv[SVEC];
    load_vec<float, SVEC>(s + n, sv);
    update(n, sv);
  }
  y = fmaf(Num<T>::to(static_cast<const T*>(p.d)[c]), x, y);
  static_cast<T*>(p.out)[static_cast<long long>(b) * p.C + c] = Num<T>::from(y * silu_f(Num<T>::to(static_cast<const T*>(p.z)[b * p.ldz + c])));
}

// lanes per channel and states per lane: as few lanes as hold the states, more of them when the channels alone leave fewer than
// four warps for each of an SM's four schedulers (a token's exponentials are too few to hide their own latency)
static void scan_split(long long channels, int N, int num_sms, int& g, int& ns) {
  g = 1;
  while (N > 16 * g) g *= 2;
  while (g < 16 && channels * g < 512ll * num_sms && (N + 2 * g - 1) / (2 * g) >= 3) g *= 2;
  ns = ((N + g - 1) / g + 3) / 4 * 4;
}

template <typename T, int NS, int G, bool STATE_ONLY>
static int scan_launch(const ScanParams& p, cudaStream_t st) {
  constexpr int CH = SC_THREADS / G;
  const size_t smem = static_cast<size_t>(SC_TB) * ((STATE_ONLY ? 1 : 2) * NS * G + (STATE_ONLY ? 2 : 3) * CH + 2 * CH) * sizeof(float) +
                      static_cast<size_t>(2) * SC_TB * (CH + (NS * G + 7) / 8 * 8) * (STATE_ONLY ? 1 : 2) * sizeof(T);
  if (smem > 44 * 1024) {      // static arrays come on top
    cudaError_t e = cudaFuncSetAttribute(selective_scan_kernel<T, NS, G, STATE_ONLY>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  selective_scan_kernel<T, NS, G, STATE_ONLY><<<dim3((p.C + CH - 1) / CH, p.B * p.nchunks), SC_THREADS, smem, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}
template <typename T, int G, bool STATE_ONLY>
static int scan_states(const ScanParams& p, int ns, cudaStream_t st) {
  if (ns == 4) return scan_launch<T, 4, G, STATE_ONLY>(p, st);
  if (ns == 8) return scan_launch<T, 8, G, STATE_ONLY>(p, st);
  if (ns == 12) return scan_launch<T, 12, G, STATE_ONLY>(p, st);
  if (ns == 16) return scan_launch<T, 16, G, STATE_ONLY>(p, st);
  return -3;
}
template <typename T, bool STATE_ONLY>
static int scan_dispatch(const ScanParams& p, int g, int ns, cudaStream_t st) {
  if (g == 1) return scan_states<T, 1, STATE_ONLY>(p, ns, st);
  if (g == 2) return scan_states<T, 2, STATE_ONLY>(p, ns, st);
  if (g == 4) return scan_states<T, 4, STATE_ONLY>(p, ns, st);
  if (g == 8) return scan_states<T, 8, STATE_ONLY>(p, ns, st);
  if (g == 16) return scan_states<T, 16, STATE_ONLY>(p, ns, st);
  return -3;
}

}  // namespace oslo

extern "C" int oslo_token_shift(const void* h, long long ldh, const void* mu, const uint8_t* keep, long long ld_keep, float* prev,
                                void* out, int B, int S, int width, int P, int dtype, cudaStream_t stream) {
  using namespace oslo;
  if (B <= 0 || S <= 0 || width <= 0) return 0;
  if (B > 65535 || (S + TS_RUN - 1) / TS_RUN > 65535) return -1;
  ShiftParams p{h, ldh, mu, keep, ld_keep, prev, out, static_cast<long long>(B) * S, S, width};
  const size_t te = dtype == OSLO_DT_FP32 ? 4 : 2;
  const bool vec = width % 4 == 0 && ldh % 4 == 0 && aligned_to(h, 4 * te) && aligned_to(mu, 4 * te) && aligned_to(out, 4 * te);
#define TS_GO(V, N)                                                                                                          \
  token_shift_kernel<T, V, N><<<dim3((width + 128 * V - 1) / (128 * V), (S + TS_RUN - 1) / TS_RUN, B), 128, 0, stream>>>(p)
  OSLO_DISPATCH_T(dtype, {
    if (P == 1) { if (vec) TS_GO(4, 1); else TS_GO(1, 1); }
    else if (P == 2) { if (vec) TS_GO(4, 2); else TS_GO(1, 2); }
    else if (P == 5) { if (vec) TS_GO(4, 5); else TS_GO(1, 5); }
    else return -3;
  });
#undef TS_GO
  return static_cast<int>(cudaGetLastError());
}

extern "C" int oslo_causal_conv(const void* x, long long ldx, const void* w, const void* bias, const uint8_t* keep,
                                long long ld_keep, float* prev, void* out, int B, int S, int C, int taps, int silu, int residual,
                                int dtype, cudaStream_t stream) {
  using namespace oslo;
  if (B <= 0 || S <= 0 || C <= 0) return 0;
  if (taps < 1 || (silu && residual)) return -1;
  ConvParams p{x, ldx, w, bias, keep, ld_keep, prev, out, S, C, taps, std::max(16, taps), silu, residual};
  const int runs = (S + p.run - 1) / p.run;
  if (B > 65535 || runs > 65535) return -1;
  const size_t te = dtype == OSLO_DT_FP32 ? 4 : 2;
  const bool vec = C % 4 == 0 && ldx % 4 == 0 && aligned_to(x, 4 * te) && aligned_to(bias, 4 * te) && aligned_to(out, 4 * te);
#define CV_GO(V, N) causal_conv_kernel<T, V, N><<<dim3((C + 128 * V - 1) / (128 * V), runs, B), 128, 0, stream>>>(p)
  OSLO_DISPATCH_T(dtype, {
    if (taps == 4 && vec) CV_GO(4, 4);
    else if (taps == 3 && vec) CV_GO(4, 3);
    else if (vec) CV_GO(4, 0);
    else CV_GO(1, 0);
  });
#undef CV_GO
  return static_cast<int>(cudaGetLastError());
}

extern "C" int oslo_scan_chunks(int B, int S, int C, int N, int num_sms) {
  using namespace oslo;
  int g, ns;
  scan_split(static_cast<long long>(B) * C, N, num_sms, g, ns);
  const int ch = SC_THREADS / g;
  const long long ctas = static_cast<long long>(B) * ((C + ch - 1) / ch);
  if (S < 128) return 1;
  // an SM's blocks share its exponential units, which fewer than four blocks do not keep busy
  int best = 1;
  double best_cost = 1e30;
  for (int n = 1; n <= S / 64 && n <= 64; ++n) {
    const double per = static_cast<double>(S) / n;
    const auto fullest = [&](long long blocks) { return static_cast<double>((blocks + num_sms - 1) / num_sms); };
    const double c3 = std::max(3.5, fullest(ctas * n)) * per;
    const double c1 = n > 1 ? std::max(3.5, fullest(ctas * (n - 1))) * per * 0.8 + 160.0 : 0.0;
    if (c3 + c1 < best_cost) { best_cost = c3 + c1; best = n; }
  }
  return best;
}

extern "C" int oslo_selective_scan(const void* x, long long ldx, const float* dt, long long lddt, const void* dt_bias,
                                   const void* a_log, const void* b, long long ldb, const void* c, long long ldc, const void* d,
                                   const void* z, long long ldz, const uint8_t* keep, long long ld_keep, float* state, void* out,
                                   float* ws, float* steps, int nchunks, int B, int S, int C, int N, int num_sms, int dtype,
                                   cudaStream_t stream) {
  using namespace oslo;
  if (B <= 0 || S <= 0 || C <= 0) return 0;
  if (N <= 0 || N > 256 || nchunks < 1 || static_cast<long long>(B) * nchunks > 65535) return -1;
  ScanParams p{};
  p.x = x; p.ldx = ldx; p.dt = dt; p.lddt = lddt; p.dt_bias = dt_bias; p.a_log = a_log; p.d = d;
  p.b = b; p.ldb = ldb; p.c = c; p.ldc = ldc; p.z = z; p.ldz = ldz; p.keep = keep; p.ld_keep = ld_keep; p.out = out;
  p.B = B; p.S = S; p.C = C; p.N = N;
  p.vec16 = C % 8 == 0 && ldx % 8 == 0 && ldz % 8 == 0 && lddt % 4 == 0 && aligned_to(x, 16) && aligned_to(z, 16) && aligned_to(dt, 16);
  p.bc16 = N % 8 == 0 && ldb % 8 == 0 && ldc % 8 == 0 && aligned_to(b, 16) && aligned_to(c, 16);
  const long long per = static_cast<long long>(C) * N;
  int rc = 0, g, ns;
  scan_split(static_cast<long long>(B) * C, N, num_sms, g, ns);
  if (nchunks == 1) {
    p.chunk = S; p.nchunks = 1; p.s_in = state; p.s_out = state; p.s_batch = per;
    OSLO_DISPATCH_T(dtype, { rc = scan_dispatch<T, false>(p, g, ns, stream); });
    return rc;
  }
  if (ws == nullptr || steps == nullptr) return -1;
  p.chunk = ((S + nchunks - 1) / nchunks + SC_TB - 1) / SC_TB * SC_TB;
  p.s_batch = per * nchunks; p.s_chunk = per;
  p.s_out = ws; p.steps = steps;
  p.nchunks = nchunks - 1;             // nobody starts from the last chunk's state
  OSLO_DISPATCH_T(dtype, { rc = scan_dispatch<T, true>(p, g, ns, stream); });
  if (rc) return rc;
  OSLO_DISPATCH_T(dtype, {
    scan_chunks_kernel<T><<<dim3(static_cast<unsigned>((per + 255) / 256), B), 256, 0, stream>>>(
        ws, steps, state, static_cast<const T*>(a_log), nchunks, C, N);
  });
  rc = static_cast<int>(cudaGetLastError());
  if (rc) return rc;
  p.nchunks = nchunks;
  p.s_in = ws; p.s_out = nullptr; p.s_end = state;
  OSLO_DISPATCH_T(dtype, { rc = scan_dispatch<T, false>(p, g, ns, stream); });
  return rc;
}

extern "C" int oslo_scan_step(const void* x, long long ldx, const void* dt, long long lddt, const void* w_dt, int rank,
                              const void* dt_bias, const void* a_log, const void* b, long long ldb, const void* c, long long ldc,
                              const void* d, const void* z, long long ldz, const uint8_t* keep, long long ld_keep, float* state,
                              void* out, int B, int C, int N, int dtype, cudaStream_t stream) {
  using namespace oslo;
  if (B <= 0 || C <= 0) return 0;
  if (N <= 0 || rank <= 0 || (B + ST_ROWS - 1) / ST_ROWS > 65535) return -1;
  ScanStepParams p{x, ldx, dt, lddt, w_dt, rank, dt_bias, a_log, d, b, c, ldb, ldc, z, ldz, keep, ld_keep, state, out, B, C, N};
  const size_t te = dtype == OSLO_DT_FP32 ? 4 : 2;
  const size_t ldd = (rank + 3) / 4 * 4;
  const bool mma = te == 2 && rank % 16 == 0 && lddt % 2 == 0 && aligned_to(w_dt, 4) && aligned_to(dt, 4);
  const size_t smem = ST_ROWS * 2 * static_cast<size_t>(N) * sizeof(float) + (mma ? 0 : ST_ROWS * ldd * sizeof(float) + ST_CH * (ldd + 4) * te);
  if (smem > 200 * 1024) return -3;
  const bool vec = rank % 4 == 0 && aligned_to(w_dt, 4 * te), svec = N % 4 == 0 && aligned_to(state, 16) && aligned_to(a_log, 4 * te);
#define SS_GO(V, SV, M)                                                                                              \
  {                                                                                                                  \
    if (smem > 40 * 1024) {                                                                                          \
      cudaError_t e = cudaFuncSetAttribute(scan_step_kernel<T, V, SV, M>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                           static_cast<int>(smem));                                                  \
      if (e != cudaSuccess) return static_cast<int>(e);                                                              \
    }                                                                                                                \
    scan_step_kernel<T, V, SV, M><<<dim3((C + ST_CH - 1) / ST_CH, (B + ST_ROWS - 1) / ST_ROWS), 256, smem, stream>>>(p); \
  }
  OSLO_DISPATCH_T(dtype, {
    if (mma && svec) SS_GO(1, 4, true)
    else if (mma) SS_GO(1, 1, true)
    else if (vec && svec) SS_GO(4, 4, false)
    else if (vec) SS_GO(4, 1, false)
    else if (svec) SS_GO(1, 4, false)
    else SS_GO(1, 1, false)
  });
#undef SS_GO
  return static_cast<int>(cudaGetLastError());
}
