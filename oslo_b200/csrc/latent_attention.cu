// Latent attention (one low-rank vector c per token is cached; every head's key W_uk c and value W_uv c come from it),
// softmax with a learned sink in the denominator, one sigmoid output gate per head.
//
// Prompts: keys and values are expanded with a GEMM. For 16-bit head sizes that the tcgen05 flash kernel takes, that
// kernel runs and sink_gate_kernel turns its (output, log-sum-exp) pair into the result:
//   out * exp(lse) / (exp(lse) + exp(sink)) * sigmoid(g) = out * sigmoid(lse - sink) * sigmoid(g).
// sink_attention_kernel covers everything else (float32, any head sizes) in 32-bit.
// Decode: keys are never expanded. latent_absorb_kernel moves W_uk to the query side (q' = W_uk^T q, 32-bit), the
// scores are q' . c, latent_decode_*_kernel accumulates sum_t p_t c_t per head over slices of the cache, and
// latent_finish_kernel merges the slices, adds the sink to the denominator, applies W_uv and the gate. All heads of a
// block share each cached vector they read.
#include <math_constants.h>

#include <algorithm>

#include "num.cuh"
#include "oslo_kernels.h"
#include "ptx.cuh"

namespace oslo {

// ------------------------------------------------------------------ prompts
// one warp per (token, head): out[row, h * vdim + j] from the flash kernel's o and lse
template <typename T>
__global__ void __launch_bounds__(256) sink_gate_kernel(const T* __restrict__ o, long long o_sb, long long o_ss, long long o_sh,
                                                        const float* __restrict__ lse, const T* __restrict__ sink,
                                                        const T* __restrict__ gate, long long ldg, T* __restrict__ out,
                                                        int B, int S, int H, int vdim) {
  const long long wid = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (wid >= static_cast<long long>(B) * S * H) return;
  const int h = static_cast<int>(wid % H);
  const long long row = wid / H;
  const long long b = row / S, s = row % S;
  const float l = lse[(b * H + h) * S + s];
  const float fac = sigmoid_f(l - Num<T>::to(sink[h])) * sigmoid_f(Num<T>::to(gate[row * ldg + h]));
  const T* src = o + b * o_sb + s * o_ss + h * o_sh;
  T* dst = out + row * (static_cast<long long>(H) * vdim) + static_cast<long long>(h) * vdim;
  if (vdim % 4 == 0) {   // the launcher checked the strides
    for (int c = lane * 4; c < vdim; c += 128) {
      float v[4];
      load_vec<T, 4>(src + c, v);
#pragma unroll
      for (int i = 0; i < 4; ++i) v[i] *= fac;
      store_vec<T, 4>(dst + c, v);
    }
  } else {
    for (int c = lane; c < vdim; c += 32) dst[c] = Num<T>::from(Num<T>::to(src[c]) * fac);
  }
}

struct SinkAttnParams {
  const void *q, *k, *v;               // row strides (b, t) and head strides in elements
  long long q_sb, q_ss, q_sh, k_sb, k_ss, k_sh, v_sb, v_ss, v_sh;
  const uint8_t* keep; long long ld_keep;   // [B, Sk], 0 = padded key
  const void* sink;
  const void* gate; long long ldg;     // row b * Sq + s
  void* out;                           // [B * Sq, H * vdim]
  int B, H, Sq, Sk, dim, vdim;
  float scale;
};

constexpr int SA_Q = 16, SA_K = 32;

// 16 queries x 32 keys per step, everything in 32-bit; 8 threads per query
template <typename T>
__global__ void __launch_bounds__(128) sink_attention_kernel(const SinkAttnParams p) {
  extern __shared__ float sa_smem[];
  const int dp = p.dim + 1, vp = p.vdim + 1;
  float* qs = sa_smem;                 // [SA_Q][dim + 1]
  float* ks = qs + SA_Q * dp;          // [SA_K][dim + 1]
  float* vs = ks + SA_K * dp;          // [SA_K][vdim + 1]
  float* os = vs + SA_K * vp;          // [SA_Q][vdim + 1]
  float* ps = os + SA_Q * vp;          // [SA_Q][SA_K + 1]
  const int b = blockIdx.z, h = blockIdx.y, q0 = blockIdx.x * SA_Q;
  const int tid = threadIdx.x, qi = tid >> 3, l8 = tid & 7;
  const int past = p.Sk - p.Sq;
  const T* q = static_cast<const T*>(p.q) + b * p.q_sb + h * p.q_sh;
  const T* k = static_cast<const T*>(p.k) + b * p.k_sb + h * p.k_sh;
  const T* v = static_cast<const T*>(p.v) + b * p.v_sb + h * p.v_sh;
  for (int e = tid; e < SA_Q * p.dim; e += 128) {
    const int r = e / p.dim, c = e % p.dim;
    qs[r * dp + c] = q0 + r < p.Sq ? Num<T>::to(q[(q0 + r) * p.q_ss + c]) : 0.f;
  }
  for (int e = tid; e < SA_Q * p.vdim; e += 128) os[(e / p.vdim) * vp + e % p.vdim] = 0.f;
  const float sink = Num<T>::to(static_cast<const T*>(p.sink)[h]);
  float m = sink, s = 1.0f;            // the sink is the first member of the denominator
  const int k_end = min(p.Sk, past + q0 + SA_Q);
  for (int k0 = 0; k0 < k_end; k0 += SA_K) {
    __syncthreads();
    for (int e = tid; e < SA_K * p.dim; e += 128) {
      const int r = e / p.dim, c = e % p.dim;
      ks[r * dp + c] = k0 + r < k_end ? Num<T>::to(k[(k0 + r) * p.k_ss + c]) : 0.f;
    }
    for (int e = tid; e < SA_K * p.vdim; e += 128) {
      const int r = e / p.vdim, c = e % p.vdim;
      vs[r * vp + c] = k0 + r < k_end ? Num<T>::to(v[(k0 + r) * p.v_ss + c]) : 0.f;
    }
    __syncthreads();
    float sc[SA_K / 8], mx = m;
#pragma unroll
    for (int u = 0; u < SA_K / 8; ++u) {
      const int kj = u * 8 + l8, pos = k0 + kj;
      float d = 0.f;
      for (int c = 0; c < p.dim; ++c) d = fmaf(qs[qi * dp + c], ks[kj * dp + c], d);
      const bool vis = pos < k_end && pos <= past + q0 + qi && (p.keep == nullptr || p.keep[b * p.ld_keep + pos]);
      sc[u] = vis ? d * p.scale : -CUDART_INF_F;
      mx = fmaxf(mx, sc[u]);
    }
#pragma unroll
    for (int off = 4; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
    const float a = expf(m - mx);      // m is finite: it starts at the sink
    float ps_sum = 0.f;
#pragma unroll
    for (int u = 0; u < SA_K / 8; ++u) {
      const float e = expf(sc[u] - mx);
      ps[qi * (SA_K + 1) + u * 8 + l8] = e;
      ps_sum += e;
    }
#pragma unroll
    for (int off = 4; off > 0; off >>= 1) ps_sum += __shfl_xor_sync(0xffffffffu, ps_sum, off);
    s = s * a + ps_sum;
    m = mx;
    __syncwarp();                      // a query's eight threads are in one warp
    for (int c = l8; c < p.vdim; c += 8) {
      float o = os[qi * vp + c] * a;
#pragma unroll 8
      for (int j = 0; j < SA_K; ++j) o = fmaf(ps[qi * (SA_K + 1) + j], vs[j * vp + c], o);
      os[qi * vp + c] = o;
    }
  }
  if (q0 + qi < p.Sq) {
    const long long row = static_cast<long long>(b) * p.Sq + q0 + qi;
    const float fac = sigmoid_f(Num<T>::to(static_cast<const T*>(p.gate)[row * p.ldg + h])) / s;
    T* out = static_cast<T*>(p.out) + row * (static_cast<long long>(p.H) * p.vdim) + static_cast<long long>(h) * p.vdim;
    for (int c = l8; c < p.vdim; c += 8) out[c] = Num<T>::from(os[qi * vp + c] * fac);
  }
}

// ------------------------------------------------------------------ decode
// block (0, b): RMS norm of the query latent; block (1, b): RMS norm of the key-value latent, written to the cache at
// position lengths[b]
template <typename T>
__global__ void __launch_bounds__(256) latent_prep_kernel(const T* __restrict__ cq, long long ldq, const T* __restrict__ wq,
                                                          int q_rank, T* __restrict__ cq_out, const T* __restrict__ ckv,
                                                          long long ldkv, const T* __restrict__ wkv, int kv_rank,
                                                          T* __restrict__ cache, const int* __restrict__ lengths, int Tmax,
                                                          float eps, int* err) {
  __shared__ float red[32];
  const int b = blockIdx.y;
  const bool is_q = blockIdx.x == 0;
  const T* x = is_q ? cq + b * ldq : ckv + b * ldkv;
  const T* w = is_q ? wq : wkv;
  const int n = is_q ? q_rank : kv_rank;
  T* out;
  if (is_q) {
    out = cq_out + static_cast<long long>(b) * q_rank;
  } else {
    const int pos = lengths[b];
    if (pos < 0 || pos >= Tmax) {      // never write outside the cache
      if (threadIdx.x == 0) OSLO_REPORT_BOUNDS(err);
      return;
    }
    out = cache + (static_cast<long long>(b) * Tmax + pos) * kv_rank;
  }
  float ss = 0.f;
  for (int c = threadIdx.x; c < n; c += blockDim.x) {
    const float v = Num<T>::to(x[c]);
    ss = fmaf(v, v, ss);
  }
  ss = block_sum(ss, red);
  const float r = 1.0f / sqrtf(ss / n + eps);
  for (int c = threadIdx.x; c < n; c += blockDim.x) out[c] = Num<T>::from(Num<T>::to(x[c]) * r * Num<T>::to(w[c]));
}

// qa[b, h, r] = scale * sum_d q[b, h * dim + d] * w_uk[h * dim + d, r]; block = (64 columns r, head, 8 rows b)
template <typename T>
__global__ void __launch_bounds__(256) latent_absorb_kernel(const T* __restrict__ q, long long ldq, const T* __restrict__ w,
                                                            long long ldw, float* __restrict__ qa, int B, int H, int dim,
                                                            int R, float scale) {
  constexpr int RB = 8, CW = 64, DG = 8;
  extern __shared__ float ab_smem[];
  float* qs = ab_smem;                 // [RB][dim]
  float* part = qs + RB * dim;         // [DG][RB][CW]
  const int h = blockIdx.y, r0 = blockIdx.x * CW, b0 = blockIdx.z * RB;
  const int nb = min(RB, B - b0);
  for (int e = threadIdx.x; e < nb * dim; e += 256) {
    const int b = e / dim, d = e % dim;
    qs[b * dim + d] = Num<T>::to(q[(b0 + b) * ldq + static_cast<long long>(h) * dim + d]) * scale;
  }
  __syncthreads();
  const int cp = threadIdx.x & 31, dg = threadIdx.x >> 5;
  const int r = r0 + cp * 2;
  float acc[RB][2];
#pragma unroll
  for (int b = 0; b < RB; ++b) acc[b][0] = acc[b][1] = 0.f;
  if (r < R) {
    const bool two = r + 1 < R;
#pragma unroll 8
    for (int d = dg; d < dim; d += DG) {
      const T* wr = w + (static_cast<long long>(h) * dim + d) * ldw + r;
      const float w0 = Num<T>::to(wr[0]), w1 = two ? Num<T>::to(wr[1]) : 0.f;
#pragma unroll
      for (int b = 0; b < RB; ++b) {
        if (b < nb) {
          const float x = qs[b * dim + d];
          acc[b][0] = fmaf(x, w0, acc[b][0]);
          acc[b][1] = fmaf(x, w1, acc[b][1]);
        }
      }
    }
  }
#pragma unroll
  for (int b = 0; b < RB; ++b) {
    part[(dg * RB + b) * CW + cp * 2] = acc[b][0];
    part[(dg * RB + b) * CW + cp * 2 + 1] = acc[b][1];
  }
  __syncthreads();
  for (int e = threadIdx.x; e < nb * CW; e += 256) {
    const int b = e / CW, c = e % CW;
    if (r0 + c >= R) continue;
    float t = 0.f;
#pragma unroll
    for (int g = 0; g < DG; ++g) t += part[(g * RB + b) * CW + c];
    qa[((static_cast<long long>(b0 + b)) * H + h) * R + r0 + c] = t;
  }
}

struct LatentDecodeParams {
  const float* qa;                     // [B, H, R], scaled
  const void* cache;                   // [B, Tmax, R]
  const int* lengths;                  // [B] valid positions
  const uint8_t* keep; long long ld_keep; int n_keep;   // [B, n_keep], 0 = padded, or nullptr
  float* ws;                           // [B, H, splits, R + 2]: sum p c, max, sum p
  int B, H, R, Tmax, splits;
  int* err;
};

constexpr int LD_HEADS = 16, LD_KEYS = 16;

// scalar version: any R, any type; block = (slice, head group, row)
template <typename T, int NR>
__global__ void __launch_bounds__(256) latent_decode_kernel(const LatentDecodeParams p) {
  extern __shared__ float ld_smem[];
  const int rp = p.R + 1;
  float* qs = ld_smem;                 // [LD_HEADS][R + 1]
  float* cs = qs + LD_HEADS * rp;      // [LD_KEYS][R + 1]
  float* sc = cs + LD_KEYS * rp;       // [LD_HEADS][LD_KEYS]
  __shared__ float resc[LD_HEADS], ms[LD_HEADS], ls[LD_HEADS];
  const int b = blockIdx.z, h0 = blockIdx.y * LD_HEADS, sp = blockIdx.x, tid = threadIdx.x;
  const int nh = min(LD_HEADS, p.H - h0);
  int len = p.lengths[b];
  if (len < 0 || len > p.Tmax) {       // a length that does not fit the cache: never read past it
    if (tid == 0) OSLO_REPORT_BOUNDS(p.err);
    len = len < 0 ? 0 : p.Tmax;
  }
  const int per = (len + p.splits - 1) / p.splits;
  const int t0 = sp * per, t1 = min(len, t0 + per);
  for (int e = tid; e < nh * p.R; e += 256)
    qs[(e / p.R) * rp + e % p.R] = p.qa[(static_cast<long long>(b) * p.H + h0) * p.R + e];
  for (int e = tid; e < (LD_HEADS - nh) * p.R; e += 256) qs[(nh + e / p.R) * rp + e % p.R] = 0.f;
  if (tid < LD_HEADS) { ms[tid] = -CUDART_INF_F; ls[tid] = 0.f; }
  float acc[NR][LD_HEADS];
#pragma unroll
  for (int j = 0; j < NR; ++j)
#pragma unroll
    for (int a = 0; a < LD_HEADS; ++a) acc[j][a] = 0.f;
  const T* c = static_cast<const T*>(p.cache) + static_cast<long long>(b) * p.Tmax * p.R;
  for (int k0 = t0; k0 < t1; k0 += LD_KEYS) {
    const int n = min(LD_KEYS, t1 - k0);
    __syncthreads();
    for (int e = tid; e < LD_KEYS * p.R; e += 256) {
      const int t = e / p.R, r = e % p.R;
      cs[t * rp + r] = t < n ? Num<T>::to(c[static_cast<long long>(k0 + t) * p.R + r]) : 0.f;
    }
    __syncthreads();
    {
      const int a = tid >> 4, t = tid & 15;
      float d = 0.f;
      for (int r = 0; r < p.R; ++r) d = fmaf(qs[a * rp + r], cs[t * rp + r], d);
      const int pos = k0 + t;
      const bool vis = t < n && (p.keep == nullptr || pos >= p.n_keep || p.keep[b * p.ld_keep + pos]);
      d = vis ? d : -CUDART_INF_F;
      float mx = d;
#pragma unroll
      for (int off = 8; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
      const float m_old = ms[a], m_new = fmaxf(m_old, mx);
      const float e = d == -CUDART_INF_F ? 0.f : expf(d - m_new);
      float s = e;
#pragma unroll
      for (int off = 8; off > 0; off >>= 1) s += __shfl_xor_sync(0xffffffffu, s, off);
      sc[a * LD_KEYS + t] = e;
      __syncwarp();
      if (t == 0) {
        const float f = m_old == -CUDART_INF_F ? 0.f : expf(m_old - m_new);
        resc[a] = f;
        ms[a] = m_new;
        ls[a] = ls[a] * f + s;
      }
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < NR; ++j) {
      const int r = tid + j * 256;
      if (r < p.R) {
#pragma unroll
        for (int a = 0; a < LD_HEADS; ++a) acc[j][a] *= resc[a];
        for (int t = 0; t < LD_KEYS; ++t) {
          const float x = cs[t * rp + r];
#pragma unroll
          for (int a = 0; a < LD_HEADS; ++a) acc[j][a] = fmaf(sc[a * LD_KEYS + t], x, acc[j][a]);
        }
      }
    }
  }
  __syncthreads();
  for (int a = 0; a < nh; ++a) {
    float* w = p.ws + ((static_cast<long long>(b) * p.H + h0 + a) * p.splits + sp) * (p.R + 2);
#pragma unroll
    for (int j = 0; j < NR; ++j) {
      const int r = tid + j * 256;
      if (r < p.R) {
        float v = 0.f;
#pragma unroll
        for (int u = 0; u < LD_HEADS; ++u) v = u == a ? acc[j][u] : v;
        w[r] = v;
      }
    }
    if (tid == 0) { w[p.R] = ms[a]; w[p.R + 1] = ls[a]; }
  }
}

// out[b, h * vdim + j] = sigmoid(g) * sum_r w_uv[h * vdim + j, r] * o[r],  o = merged slices / (sum + exp(sink))
template <typename T, int VEC>
__global__ void __launch_bounds__(256) latent_finish_kernel(const float* __restrict__ ws, const T* __restrict__ w, long long ldw,
                                                            const T* __restrict__ sink, const T* __restrict__ gate,
                                                            long long ldg, T* __restrict__ out, int H, int R, int vdim,
                                                            int splits, int rows_per_block) {
  extern __shared__ float fin_smem[];   // [R] then [splits] weights
  float* o = fin_smem;
  float* wt = fin_smem + R;
  const int h = blockIdx.y, b = blockIdx.z;
  const float* base = ws + (static_cast<long long>(b) * H + h) * splits * (R + 2);
  const float snk = Num<T>::to(sink[h]);
  float m = snk;
  for (int s = 0; s < splits; ++s) m = fmaxf(m, base[static_cast<long long>(s) * (R + 2) + R]);
  float tot = expf(snk - m);
  for (int s = 0; s < splits; ++s) {
    const float ms = base[static_cast<long long>(s) * (R + 2) + R];
    const float f = ms == -CUDART_INF_F ? 0.f : expf(ms - m);
    tot += f * base[static_cast<long long>(s) * (R + 2) + R + 1];
    if (threadIdx.x == 0) wt[s] = f;
  }
  __syncthreads();
  const float inv = sigmoid_f(Num<T>::to(gate[b * ldg + h])) / tot;
  for (int r = threadIdx.x; r < R; r += blockDim.x) {
    float v = 0.f;
    for (int s = 0; s < splits; ++s)
      if (wt[s] != 0.f) v = fmaf(wt[s], base[static_cast<long long>(s) * (R + 2) + r], v);
    o[r] = v * inv;
  }
  __syncthreads();
  const int lane = threadIdx.x & 31;
  const int j1 = min(vdim, (static_cast<int>(blockIdx.x) + 1) * rows_per_block);
  for (int j = blockIdx.x * rows_per_block + (threadIdx.x >> 5); j < j1; j += blockDim.x >> 5) {
    const float d = warp_dot<T, VEC>(w + (static_cast<long long>(h) * vdim + j) * ldw, o, R, lane);
    if (lane == 0) out[(static_cast<long long>(b) * H + h) * vdim + j] = Num<T>::from(d);
  }
}

static int set_smem(const void* fn, size_t bytes) {
  if (bytes <= 48 * 1024) return 0;
  if (bytes > 227 * 1024) return -3;
  return static_cast<int>(cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes)));
}

}  // namespace oslo

extern "C" int oslo_sink_gate(const void* o, long long o_sb, long long o_ss, long long o_sh, const float* lse, const void* sink,
                              const void* gate, long long ldg, void* out, int B, int S, int H, int vdim, int dtype,
                              cudaStream_t stream) {
  using namespace oslo;
  const long long warps = static_cast<long long>(B) * S * H;
  if (warps <= 0) return 0;
  const size_t te = dtype == OSLO_DT_FP32 ? 4 : 2;
  if (vdim % 4 == 0 && ((o_sb | o_ss | o_sh) % 4 || !aligned_to(o, 4 * te) || !aligned_to(out, 4 * te))) return -4;
  OSLO_DISPATCH_T(dtype, {
    sink_gate_kernel<T><<<static_cast<unsigned>((warps + 7) / 8), 256, 0, stream>>>(
        static_cast<const T*>(o), o_sb, o_ss, o_sh, lse, static_cast<const T*>(sink), static_cast<const T*>(gate), ldg,
        static_cast<T*>(out), B, S, H, vdim);
  });
  return static_cast<int>(cudaGetLastError());
}

extern "C" int oslo_sink_attention(const void* q, long long q_sb, long long q_ss, long long q_sh, const void* k, long long k_sb,
                                   long long k_ss, long long k_sh, const void* v, long long v_sb, long long v_ss,
                                   long long v_sh, const uint8_t* keep, long long ld_keep, const void* sink, const void* gate,
                                   long long ldg, void* out, int B, int H, int Sq, int Sk, int dim, int vdim, float scale,
                                   int dtype, cudaStream_t stream) {
  using namespace oslo;
  if (B <= 0 || H <= 0 || Sq <= 0) return 0;
  if (Sk < Sq || B > 65535 || H > 65535) return -1;
  SinkAttnParams p{q, k, v, q_sb, q_ss, q_sh, k_sb, k_ss, k_sh, v_sb, v_ss, v_sh, keep, ld_keep, sink, gate, ldg, out,
                   B, H, Sq, Sk, dim, vdim, scale};
  const size_t smem = (static_cast<size_t>(SA_Q + SA_K) * (dim + 1 + vdim + 1) + SA_Q * (SA_K + 1)) * sizeof(float);
  dim3 grid((Sq + SA_Q - 1) / SA_Q, H, B);
  OSLO_DISPATCH_T(dtype, {
    const int rc = set_smem(reinterpret_cast<const void*>(&sink_attention_kernel<T>), smem);
    if (rc) return rc;
    sink_attention_kernel<T><<<grid, 128, smem, stream>>>(p);
  });
  return static_cast<int>(cudaGetLastError());
}

extern "C" int oslo_latent_prep(const void* cq, long long ldq, const void* wq, int q_rank, void* cq_out, const void* ckv,
                                long long ldkv, const void* wkv, int kv_rank, void* cache, const int* lengths, int Tmax,
                                float eps, int B, int dtype, int* err_word, cudaStream_t stream) {
  using namespace oslo;
  if (B <= 0) return 0;
  OSLO_DISPATCH_T(dtype, {
    latent_prep_kernel<T><<<dim3(ckv ? 2 : 1, B), 256, 0, stream>>>(
        static_cast<const T*>(cq), ldq, static_cast<const T*>(wq), q_rank, static_cast<T*>(cq_out), static_cast<const T*>(ckv),
        ldkv, static_cast<const T*>(wkv), kv_rank, static_cast<T*>(cache), lengths, Tmax, eps, err_word);
  });
  return static_cast<int>(cudaGetLastError());
}

extern "C" int oslo_latent_decode(const void* q, long long ldq, const void* w_uk, long long ldk, const void* w_uv, long long ldv,
                                  const void* cache, const int* lengths, const uint8_t* keep, long long ld_keep, int n_keep,
                                  const void* sink, const void* gate, long long ldg, float* qa, float* ws, void* out, int B,
                                  int H, int dim, int vdim, int R, int Tmax, int splits, float scale, int dtype, int* err_word,
                                  cudaStream_t stream) {
  using namespace oslo;
  if (B <= 0 || H <= 0) return 0;
  if (R <= 0 || R > 1024 || splits < 1 || B > 65535) return -1;
  LatentDecodeParams p{qa, cache, lengths, keep, ld_keep, n_keep, ws, B, H, R, Tmax, splits, err_word};
  const size_t te = dtype == OSLO_DT_FP32 ? 4 : 2;
  const size_t ab_smem = (8 * static_cast<size_t>(dim) + 8 * 8 * 64) * sizeof(float);
  const size_t ld_smem = (static_cast<size_t>(LD_HEADS + LD_KEYS) * (R + 1) + LD_HEADS * LD_KEYS) * sizeof(float);
  const size_t fin_smem = static_cast<size_t>(R + splits) * sizeof(float);
  dim3 grid(splits, (H + LD_HEADS - 1) / LD_HEADS, B);
#define LD_GO(NR)                                                                             \
  {                                                                                           \
    rc = set_smem(reinterpret_cast<const void*>(&latent_decode_kernel<T, NR>), ld_smem);      \
    if (rc) return rc;                                                                        \
    latent_decode_kernel<T, NR><<<grid, 256, ld_smem, stream>>>(p);                           \
  }
  OSLO_DISPATCH_T(dtype, {
    int rc = set_smem(reinterpret_cast<const void*>(&latent_absorb_kernel<T>), ab_smem);
    if (rc) return rc;
    latent_absorb_kernel<T><<<dim3((R + 63) / 64, H, (B + 7) / 8), 256, ab_smem, stream>>>(
        static_cast<const T*>(q), ldq, static_cast<const T*>(w_uk), ldk, qa, B, H, dim, R, scale);
    if (R <= 256) LD_GO(1)
    else if (R <= 512) LD_GO(2)
    else LD_GO(4)
    int parts = 1;                     // value rows of a head over several blocks while the GPU has room
    while (parts < 8 && static_cast<long long>(B) * H * parts < 148 && vdim / (2 * parts) >= 8) parts *= 2;
    const int rpb = (vdim + parts - 1) / parts;
    const bool vec = R % 4 == 0 && ldv % 4 == 0 && aligned_to(w_uv, 4 * te);
    if (vec)
      latent_finish_kernel<T, 4><<<dim3(parts, H, B), 256, fin_smem, stream>>>(
          ws, static_cast<const T*>(w_uv), ldv, static_cast<const T*>(sink), static_cast<const T*>(gate), ldg,
          static_cast<T*>(out), H, R, vdim, splits, rpb);
    else
      latent_finish_kernel<T, 1><<<dim3(parts, H, B), 256, fin_smem, stream>>>(
          ws, static_cast<const T*>(w_uv), ldv, static_cast<const T*>(sink), static_cast<const T*>(gate), ldg,
          static_cast<T*>(out), H, R, vdim, splits, rpb);
  });
#undef LD_GO
  return static_cast<int>(cudaGetLastError());
}
