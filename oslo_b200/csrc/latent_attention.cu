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

// 16-bit version on the tensor cores for R % 16 == 0: the 16 heads of a group are the 16 rows of an m16n8k16 tile, so the
// cache streams through shared memory once for all of them. 8 warps; per KT cached vectors:
//   scores  the warps cover the KT / 8 key columns (and halves of R when KT = 32); q' is split into two 16-bit terms
//   softmax warp w owns heads 2 w and 2 w + 1 (running max and sum in registers), P is stored as 16-bit
//   output  a warp owns every eighth pair of 8-column blocks of R; the cached vectors are read transposed
// The next KT vectors are fetched with cp.async meanwhile.
template <typename T> struct MmaT;
template <> struct MmaT<__nv_bfloat16> {
  static __device__ __forceinline__ void mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
  }
};
template <> struct MmaT<__half> {
  static __device__ __forceinline__ void mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
  }
};
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm2(uint32_t addr, uint32_t& r0, uint32_t& r1) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void ldsm4_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}

template <typename T, int KT, int NP>   // KT cached vectors per step (64 or 32), NP pairs of 8-column blocks per warp
__global__ void __launch_bounds__(256, 1) latent_decode_mma_kernel(const LatentDecodeParams p) {
  constexpr int KS = KT == 64 ? 1 : 2;  // slices of R in the score product
  constexpr int PP = KT + 8;            // padded row of P
  extern __shared__ __align__(16) uint8_t lm_smem[];
  const int rp = p.R + 8;               // padded row: 16-byte aligned, conflict-free ldmatrix
  T* q_hi = reinterpret_cast<T*>(lm_smem);          // [16][rp]
  T* q_lo = q_hi + 16 * rp;
  T* cs = q_lo + 16 * rp;                           // [2][KT][rp]
  T* ps = cs + 2 * KT * rp;                         // [16][PP]
  float* ss = reinterpret_cast<float*>(ps + 16 * PP);   // [KS][16][KT + 1]
  float* fac = ss + KS * 16 * (KT + 1);             // [16]
  const int b = blockIdx.z, h0 = blockIdx.y * LD_HEADS, sp = blockIdx.x, tid = threadIdx.x;
  const int warp = tid >> 5, lane = tid & 31;
  const int nh = min(LD_HEADS, p.H - h0);
  int len = p.lengths[b];
  if (len < 0 || len > p.Tmax) {       // a length that does not fit the cache: never read past it
    if (tid == 0) OSLO_REPORT_BOUNDS(p.err);
    len = len < 0 ? 0 : p.Tmax;
  }
  const int tiles = (len + KT - 1) / KT, per = (tiles + p.splits - 1) / p.splits * KT;
  const int t0 = sp * per, t1 = min(len, t0 + per);
  const T* c = static_cast<const T*>(p.cache) + static_cast<long long>(b) * p.Tmax * p.R;
  const int vr = p.R / 8;              // 16-byte pieces of a cached vector
  auto fetch = [&](int k0, int buf) {
    T* dst = cs + static_cast<size_t>(buf) * KT * rp;
    for (int e = tid; e < KT * vr; e += 256) {
      const int t = e / vr, v = e - t * vr;
      const uint32_t d32 = smem_u32(dst + t * rp + v * 8);
      const bool in = k0 + t < t1;     // rows past the slice are zero-filled (source size 0)
      const T* src = c + static_cast<long long>(in ? k0 + t : 0) * p.R + v * 8;
      const int bytes = in ? 16 : 0;
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d32), "l"(src), "r"(bytes) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (t0 < t1) fetch(t0, 0);
  for (int e = tid; e < 16 * p.R; e += 256) {
    const int a = e / p.R, r = e - a * p.R;
    const float x = a < nh ? p.qa[(static_cast<long long>(b) * p.H + h0 + a) * p.R + r] : 0.f;
    const T hi = Num<T>::from(x);
    q_hi[a * rp + r] = hi;
    q_lo[a * rp + r] = Num<T>::from(x - Num<T>::to(hi));
  }
  float acc[NP][2][4];
#pragma unroll
  for (int j = 0; j < NP; ++j)
#pragma unroll
    for (int u = 0; u < 2; ++u)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[j][u][i] = 0.f;
  float m_run[2] = {-CUDART_INF_F, -CUDART_INF_F}, l_run[2] = {0.f, 0.f};
  const int arow = lane & 15, acol = (lane >> 4) * 8;      // ldmatrix.x4 source of an A fragment
  for (int k0 = t0, it = 0; k0 < t1; k0 += KT, ++it) {
    const int buf = it & 1;
    if (k0 + KT < t1) {                                    // the other buffer was last read before the closing barrier
      fetch(k0 + KT, buf ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const T* ct = cs + static_cast<size_t>(buf) * KT * rp;
    {
      const int kg = warp % (KT / 8), ks = warp / (KT / 8);
      const int n16 = p.R / 16, s_begin = ks * n16 / KS, s_end = (ks + 1) * n16 / KS;
      float d[4] = {0.f, 0.f, 0.f, 0.f}, e[4] = {0.f, 0.f, 0.f, 0.f};
      for (int s = s_begin; s < s_end; ++s) {
        uint32_t ah[4], al[4], b0, b1;
        ldsm4(smem_u32(q_hi + arow * rp + s * 16 + acol), ah);
        ldsm4(smem_u32(q_lo + arow * rp + s * 16 + acol), al);
        ldsm2(smem_u32(ct + (kg * 8 + (lane & 7)) * rp + s * 16 + ((lane >> 3) & 1) * 8), b0, b1);
        MmaT<T>::mma(d, ah, b0, b1);
        MmaT<T>::mma(e, al, b0, b1);
      }
      float* o = ss + ks * 16 * (KT + 1) + (lane >> 2) * (KT + 1) + kg * 8 + (lane & 3) * 2;
      o[0] = d[0] + e[0]; o[1] = d[1] + e[1];
      o[8 * (KT + 1)] = d[2] + e[2]; o[8 * (KT + 1) + 1] = d[3] + e[3];
    }
    __syncthreads();
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int a = warp * 2 + u;
      float x[KT / 32], mx = m_run[u];
#pragma unroll
      for (int i = 0; i < KT / 32; ++i) {
        const int t = lane + 32 * i, pos = k0 + t;
        float v = ss[a * (KT + 1) + t];
        if (KS == 2) v += ss[16 * (KT + 1) + a * (KT + 1) + t];
        const bool vis = pos < t1 && (p.keep == nullptr || pos >= p.n_keep || p.keep[b * p.ld_keep + pos]);
        x[i] = vis ? v : -CUDART_INF_F;
        mx = fmaxf(mx, x[i]);
      }
#pragma unroll
      for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < KT / 32; ++i) {
        const float pr = x[i] == -CUDART_INF_F ? 0.f : expf(x[i] - mx);
        sum += pr;
        ps[a * PP + lane + 32 * i] = Num<T>::from(pr);
      }
      sum = warp_sum(sum);
      const float f = m_run[u] == -CUDART_INF_F ? 0.f : expf(m_run[u] - mx);
      l_run[u] = l_run[u] * f + sum;
      m_run[u] = mx;
      if (lane == 0) fac[a] = f;
    }
    __syncthreads();
    const float f0 = fac[lane >> 2], f1 = fac[(lane >> 2) + 8];
#pragma unroll
    for (int j = 0; j < NP; ++j)
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        acc[j][u][0] *= f0; acc[j][u][1] *= f0; acc[j][u][2] *= f1; acc[j][u][3] *= f1;
      }
#pragma unroll
    for (int s = 0; s < KT / 16; ++s) {
      uint32_t a[4];
      ldsm4(smem_u32(ps + arow * PP + s * 16 + acol), a);
#pragma unroll
      for (int j = 0; j < NP; ++j) {
        const int col = (warp + 8 * j) * 16;
        if (col < p.R) {                                   // uniform over the warp
          uint32_t bb[4];
          ldsm4_t(smem_u32(ct + (s * 16 + (lane & 15)) * rp + col + (lane >> 4) * 8), bb);
          MmaT<T>::mma(acc[j][0], a, bb[0], bb[1]);
          MmaT<T>::mma(acc[j][1], a, bb[2], bb[3]);
        }
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int j = 0; j < NP; ++j) {
    const int col = (warp + 8 * j) * 16;
    if (col >= p.R) continue;
#pragma unroll
    for (int u = 0; u < 2; ++u)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int a = (lane >> 2) + 8 * hf;
        if (a < nh) {
          float* w = p.ws + ((static_cast<long long>(b) * p.H + h0 + a) * p.splits + sp) * (p.R + 2) + col + u * 8 + (lane & 3) * 2;
          w[0] = acc[j][u][hf * 2];
          w[1] = acc[j][u][hf * 2 + 1];
        }
      }
  }
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    const int a = warp * 2 + u;
    if (lane == 0 && a < nh) {
      float* w = p.ws + ((static_cast<long long>(b) * p.H + h0 + a) * p.splits + sp) * (p.R + 2) + p.R;
      w[0] = m_run[u];
      w[1] = l_run[u];
    }
  }
}
static size_t latent_mma_smem(int R, int kt) {
  const size_t rp = R + 8;
  return (32 * rp + 2 * kt * rp + 16 * (kt + 8)) * 2 + ((kt == 64 ? 1 : 2) * 16 * (kt + 1) + 16) * sizeof(float);
}

// out[b, h * vdim + j] = sigmoid(g) * sum_r w_uv[h * vdim + j, r] * o[r],  o = merged slices / (sum + exp(sink))
// for NB rows b per block, so that W_uv is read once for all of them
template <typename T, int VEC, int NB>
__global__ void __launch_bounds__(256) latent_finish_kernel(const float* __restrict__ ws, const T* __restrict__ w, long long ldw,
                                                            const T* __restrict__ sink, const T* __restrict__ gate,
                                                            long long ldg, T* __restrict__ out, int B, int H, int R, int vdim,
                                                            int splits, int rows_per_block) {
  extern __shared__ float fin_smem[];   // [NB][R] then [NB][splits] weights
  float* o = fin_smem;
  float* wt = fin_smem + NB * R;
  const int h = blockIdx.y, b0 = blockIdx.z * NB, nb = min(NB, B - b0);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const float snk = Num<T>::to(sink[h]);
  for (int i = warp; i < nb; i += 8) {  // slice weights of a row, already divided by the denominator and gated
    const float* st = ws + (static_cast<long long>(b0 + i) * H + h) * splits * (R + 2) + R;
    float m = snk;
    for (int s = lane; s < splits; s += 32) m = fmaxf(m, st[static_cast<long long>(s) * (R + 2)]);
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, off));
    float tot = 0.f;
    for (int s = lane; s < splits; s += 32) {
      const float ms = st[static_cast<long long>(s) * (R + 2)];
      const float f = ms == -CUDART_INF_F ? 0.f : expf(ms - m);
      tot += f * st[static_cast<long long>(s) * (R + 2) + 1];
      wt[i * splits + s] = f;
    }
    tot = warp_sum(tot) + expf(snk - m);
    const float inv = sigmoid_f(Num<T>::to(gate[(b0 + i) * ldg + h])) / tot;
    for (int s = lane; s < splits; s += 32) wt[i * splits + s] *= inv;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < nb * R; e += blockDim.x) {
    const int i = e / R, r = e - i * R;
    const float* base = ws + (static_cast<long long>(b0 + i) * H + h) * splits * (R + 2) + r;
    float v = 0.f;
#pragma unroll 8
    for (int s = 0; s < splits; ++s) v = fmaf(wt[i * splits + s], base[static_cast<long long>(s) * (R + 2)], v);
    o[i * R + r] = v;
  }
  __syncthreads();
  const int j1 = min(vdim, (static_cast<int>(blockIdx.x) + 1) * rows_per_block);
  for (int j = blockIdx.x * rows_per_block + warp; j < j1; j += 8) {
    const T* wr = w + (static_cast<long long>(h) * vdim + j) * ldw;
    float acc[NB];
#pragma unroll
    for (int i = 0; i < NB; ++i) acc[i] = 0.f;
    for (int k = lane * VEC; k < R; k += 32 * VEC) {
      float x[VEC];
      load_vec<T, VEC>(wr + k, x);
#pragma unroll
      for (int i = 0; i < NB; ++i)
        if (i < nb) {
#pragma unroll
          for (int u = 0; u < VEC; ++u) acc[i] = fmaf(x[u], o[i * R + k + u], acc[i]);
        }
    }
#pragma unroll
    for (int i = 0; i < NB; ++i) {
      const float d = warp_sum(acc[i]);
      if (lane == 0 && i < nb) out[(static_cast<long long>(b0 + i) * H + h) * vdim + j] = Num<T>::from(d);
    }
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

namespace oslo {

template <typename T>
static int latent_scan(const LatentDecodeParams& p, int use_mma, cudaStream_t st) {
  dim3 grid(p.splits, (p.H + LD_HEADS - 1) / LD_HEADS, p.B);
  if constexpr (sizeof(T) == 2) {
    if (use_mma) {
      const int kt = p.R <= 512 ? 64 : 32, np = (p.R + 127) / 128;
      const size_t smem = latent_mma_smem(p.R, kt);
#define LM_GO(KT, NP)                                                                                   \
  {                                                                                                     \
    const int rc = set_smem(reinterpret_cast<const void*>(&latent_decode_mma_kernel<T, KT, NP>), smem); \
    if (rc) return rc;                                                                                  \
    latent_decode_mma_kernel<T, KT, NP><<<grid, 256, smem, st>>>(p);                                    \
    return static_cast<int>(cudaGetLastError());                                                        \
  }
      if (np == 1) LM_GO(64, 1)
      if (np == 2) LM_GO(64, 2)
      if (np <= 4) LM_GO(64, 4)
      LM_GO(32, 8)
#undef LM_GO
    }
  }
  const size_t smem = (static_cast<size_t>(LD_HEADS + LD_KEYS) * (p.R + 1) + LD_HEADS * LD_KEYS) * sizeof(float);
#define LD_GO(NR)                                                                             \
  {                                                                                           \
    const int rc = set_smem(reinterpret_cast<const void*>(&latent_decode_kernel<T, NR>), smem); \
    if (rc) return rc;                                                                        \
    latent_decode_kernel<T, NR><<<grid, 256, smem, st>>>(p);                                  \
  }
  if (p.R <= 256) LD_GO(1)
  else if (p.R <= 512) LD_GO(2)
  else LD_GO(4)
#undef LD_GO
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int VEC>
static int latent_finish(const LatentDecodeParams& p, const void* w_uv, long long ldv, const void* sink, const void* gate,
                         long long ldg, void* out, int vdim, int num_sms, cudaStream_t st) {
  const int nb = p.B >= 8 ? 8 : (p.B >= 2 ? 2 : 1), zb = (p.B + nb - 1) / nb;
  int parts = 1;                       // value rows of a head over several blocks while the GPU has room
  while (parts < 16 && static_cast<long long>(zb) * p.H * parts < num_sms && vdim / (2 * parts) >= 8) parts *= 2;
  const int rpb = (vdim + parts - 1) / parts;
  const size_t smem = static_cast<size_t>(nb) * (p.R + p.splits) * sizeof(float);
  dim3 grid(parts, p.H, zb);
#define FIN_GO(NB)                                                                                                    \
  latent_finish_kernel<T, VEC, NB><<<grid, 256, smem, st>>>(p.ws, static_cast<const T*>(w_uv), ldv, static_cast<const T*>(sink), \
                                                            static_cast<const T*>(gate), ldg, static_cast<T*>(out), p.B, p.H, p.R, \
                                                            vdim, p.splits, rpb)
  if (nb == 8) FIN_GO(8);
  else if (nb == 2) FIN_GO(2);
  else FIN_GO(1);
#undef FIN_GO
  return static_cast<int>(cudaGetLastError());
}

}  // namespace oslo

// slices of the cache per (row, head group): fewest waves of blocks, then the least work per block
extern "C" int oslo_latent_splits(int B, int H, int T, int R, int num_sms) {
  const int groups = (H + oslo::LD_HEADS - 1) / oslo::LD_HEADS, kt = R <= 512 ? 64 : 32, tiles = (T + kt - 1) / kt;
  int best = 1;
  double best_cost = 1e30;
  for (int s = 1; s <= 32 && s <= tiles; ++s) {
    const long long waves = (static_cast<long long>(B) * groups * s + num_sms - 1) / num_sms;
    const double cost = static_cast<double>(waves) * ((tiles + s - 1) / s + 1.5) + 0.05 * s;   // set-up and merge of a slice
    if (cost < best_cost) { best_cost = cost; best = s; }
  }
  return best;
}

extern "C" int oslo_latent_decode(const void* q, long long ldq, const void* w_uk, long long ldk, const void* w_uv, long long ldv,
                                  const void* cache, const int* lengths, const uint8_t* keep, long long ld_keep, int n_keep,
                                  const void* sink, const void* gate, long long ldg, float* qa, float* ws, void* out, int B,
                                  int H, int dim, int vdim, int R, int Tmax, int splits, float scale, int num_sms, int dtype,
                                  int* err_word, cudaStream_t stream) {
  using namespace oslo;
  if (B <= 0 || H <= 0) return 0;
  if (R <= 0 || R > 1024 || splits < 1 || splits > 64 || B > 65535 || H > 65535) return -1;
  LatentDecodeParams p{qa, cache, lengths, keep, ld_keep, n_keep, ws, B, H, R, Tmax, splits, err_word};
  const size_t te = dtype == OSLO_DT_FP32 ? 4 : 2;
  const size_t ab_smem = (8 * static_cast<size_t>(dim) + 8 * 8 * 64) * sizeof(float);
  OSLO_DISPATCH_T(dtype, {
    int rc = set_smem(reinterpret_cast<const void*>(&latent_absorb_kernel<T>), ab_smem);
    if (rc) return rc;
    latent_absorb_kernel<T><<<dim3((R + 63) / 64, H, (B + 7) / 8), 256, ab_smem, stream>>>(
        static_cast<const T*>(q), ldq, static_cast<const T*>(w_uk), ldk, qa, B, H, dim, R, scale);
    rc = latent_scan<T>(p, R % 16 == 0 && aligned_to(cache, 16), stream);
    if (rc) return rc;
    const bool vec = R % 4 == 0 && ldv % 4 == 0 && aligned_to(w_uv, 4 * te);
    return vec ? latent_finish<T, 4>(p, w_uv, ldv, sink, gate, ldg, out, vdim, num_sms, stream)
               : latent_finish<T, 1>(p, w_uv, ldv, sink, gate, ldg, out, vdim, num_sms, stream);
  });
  return -2;
}
