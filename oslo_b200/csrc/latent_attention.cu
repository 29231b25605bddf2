// Latent attention (one low-rank vector c per token is cached; every head's key W_uk c and value W_uv c come from it), optionally
// with a rotated key part that all heads share (cached behind c), a learned sink in the softmax denominator, sigmoid output
// gates per head or per element.
//
// Prompts: keys and values are expanded with a GEMM. For 16-bit head sizes that the tcgen05 flash kernel takes, that
// kernel runs and sink_gate_kernel turns its (output, log-sum-exp) pair into the result:
//   out * exp(lse) / (exp(lse) + exp(sink)) * sigmoid(g) = out * sigmoid(lse - sink) * sigmoid(g).
// sink_attention_kernel covers everything else (float32, any head sizes) in 32-bit.
// Decode: keys are never expanded. latent_absorb_kernel moves W_uk to the query side (q' = W_uk^T q, 32-bit) and rotates the
// query's own rotated part, which follows q'; the scores are q' . (c and what is cached behind it), latent_decode_*_kernel accumulates sum_t p_t c_t per head over slices of the cache, and
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
  const void* gate; long long ldg;     // row b * Sq + s; nullptr: no output gate
  void* out;                           // [B * Sq, H * vdim]
  int B, H, G, KG, Sq, Sk, dim, vdim;  // query head h reads key head h / (H / KG) and value head h / (H / G)
  float scale, softcap;                // softcap > 0: scores become softcap * tanh(score / softcap)
  int window, keep_first;              // window > 0: the last `window` keys, and the first keep_first after lead[b]
  const int* lead;                     // [B] padding ahead of the sequence, or nullptr
  int gate_wide;                       // the gate has a column per output column
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
  const T* k = static_cast<const T*>(p.k) + b * p.k_sb + h / (p.H / p.KG) * p.k_sh;
  const T* v = static_cast<const T*>(p.v) + b * p.v_sb + h / (p.H / p.G) * p.v_sh;
  for (int e = tid; e < SA_Q * p.dim; e += 128) {
    const int r = e / p.dim, c = e % p.dim;
    qs[r * dp + c] = q0 + r < p.Sq ? Num<T>::to(q[(q0 + r) * p.q_ss + c]) : 0.f;
  }
  for (int e = tid; e < SA_Q * p.vdim; e += 128) os[(e / p.vdim) * vp + e % p.vdim] = 0.f;
  // the sink is the first member of the denominator
  float m = p.sink ? Num<T>::to(static_cast<const T*>(p.sink)[h]) : -CUDART_INF_F, s = p.sink ? 1.0f : 0.f;
  const int k_end = min(p.Sk, past + q0 + SA_Q);
  const int kept = p.window > 0 ? (p.lead ? p.lead[b] : 0) + p.keep_first : 0;     // keys before this one are in every window
  const int near = p.window > 0 ? past + q0 - p.window + 1 : 0;                    // no window of this block starts earlier
  for (int k0 = 0; k0 < k_end; k0 += SA_K) {
    if (k0 + SA_K <= near && k0 >= kept) continue;     // uniform over the block
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
      const bool in = p.window <= 0 || past + q0 + qi - pos < p.window || pos < kept;
      const bool vis = in && pos < k_end && pos <= past + q0 + qi && (p.keep == nullptr || p.keep[b * p.ld_keep + pos]);
      d *= p.scale;
      if (p.softcap > 0.f) d = p.softcap * tanhf(d / p.softcap);
      sc[u] = vis ? d : -CUDART_INF_F;
      mx = fmaxf(mx, sc[u]);
    }
#pragma unroll
    for (int off = 4; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
    const float base = mx == -CUDART_INF_F ? 0.f : mx; // nothing seen yet: every term is exp(-inf) = 0
    const float a = expf(m - base);
    float ps_sum = 0.f;
#pragma unroll
    for (int u = 0; u < SA_K / 8; ++u) {
      const float e = expf(sc[u] - base);
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
    const T* gate = static_cast<const T*>(p.gate) + (p.gate ? row * p.ldg : 0);
    float fac = s > 0.f ? 1.0f / s : 0.f;              // a padded query may see nothing
    if (p.gate && !p.gate_wide) fac *= sigmoid_f(Num<T>::to(gate[h]));
    T* out = static_cast<T*>(p.out) + row * (static_cast<long long>(p.H) * p.vdim) + static_cast<long long>(h) * p.vdim;
    for (int c = l8; c < p.vdim; c += 8) {
      const float g = p.gate && p.gate_wide ? sigmoid_f(Num<T>::to(gate[static_cast<long long>(h) * p.vdim + c])) : 1.0f;
      out[c] = Num<T>::from(os[qi * vp + c] * fac * g);
    }
  }
}

// ------------------------------------------------------------------ decode
// the pair (x, y) turned by the angle a
__device__ __forceinline__ void turn(float a, float& x, float& y) {
  float sn, cs;
  sincosf(a, &sn, &cs);
  const float u = x * cs - y * sn;
  y = y * cs + x * sn;
  x = u;
}

struct LatentPrepParams {
  const void *cq, *wq; long long ldq; int q_rank;
  void* cq_out;
  const void *ckv, *wkv; long long ldkv; int kv_rank, rot;
  void* cache;                         // [B, Tmax, kv_rank + rot]
  void* c_out;                         // [B * S, kv_rank] or nullptr
  const int* lengths;
  const long long* pos; long long pos_sb, pos_ss;
  const float* freq;                   // [rot / 2]
  int S, Tmax;
  float eps;
  int* err;
};

// block (0, row b * S + t): RMS norm of the query latent; block (1, row): RMS norm of the key-value latent and rotation of the key
// part behind it, written to the cache at position lengths[b] + t. VEC 4: rows and sizes are aligned to four elements
template <typename T, int VEC>
__global__ void __launch_bounds__(256) latent_prep_kernel(const LatentPrepParams p) {
  __shared__ float red[32];
  const long long row = blockIdx.x;
  const bool is_q = blockIdx.y == 0;
  const T* x = is_q ? static_cast<const T*>(p.cq) + row * p.ldq : static_cast<const T*>(p.ckv) + row * p.ldkv;
  const T* w = static_cast<const T*>(is_q ? p.wq : p.wkv);
  const int n = is_q ? p.q_rank : p.kv_rank;
  T *out, *again = nullptr;
  if (is_q) {
    out = static_cast<T*>(p.cq_out) + row * p.q_rank;
  } else {
    const long long b = row / p.S, t = row - b * p.S;
    const long long at = p.lengths[b] + t;
    if (at < 0 || at >= p.Tmax) {      // never write outside the cache
      if (threadIdx.x == 0) OSLO_REPORT_BOUNDS(p.err);
      return;
    }
    out = static_cast<T*>(p.cache) + (b * p.Tmax + at) * (p.kv_rank + p.rot);
    if (p.c_out) again = static_cast<T*>(p.c_out) + row * p.kv_rank;
    const int half = p.rot / 2;
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
      float u = Num<T>::to(x[n + i]), v = Num<T>::to(x[n + half + i]);
      turn(static_cast<float>(p.pos[b * p.pos_sb + t * p.pos_ss]) * p.freq[i], u, v);
      out[n + i] = Num<T>::from(u);
      out[n + half + i] = Num<T>::from(v);
    }
  }
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < n; c += blockDim.x * VEC) {
    float v[VEC];
    load_vec<T, VEC>(x + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss = fmaf(v[i], v[i], ss);
  }
  ss = block_sum(ss, red);
  const float r = 1.0f / sqrtf(ss / n + p.eps);
  for (int c = threadIdx.x * VEC; c < n; c += blockDim.x * VEC) {
    float v[VEC], g[VEC];
    load_vec<T, VEC>(x + c, v);
    load_vec<T, VEC>(w + c, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] *= r * g[i];
    store_vec<T, VEC>(out + c, v);
    if (again) store_vec<T, VEC>(again + c, v);
  }
}

// in place: a thread turns VEC neighbouring pairs of one head's last rot dims; block = (rows, heads x groups of pairs)
template <typename T, int VEC>
__global__ void __launch_bounds__(256) rotate_halves_kernel(T* __restrict__ q, const long long* __restrict__ pos, long long pos_sb,
                                                            long long pos_ss, const float* __restrict__ freq, int S, int H, int dim,
                                                            int rot, int per_head) {
  const int half = rot / 2;
  const long long row = blockIdx.x, b = row / S, t = row - b * S;
  const float at = static_cast<float>(pos[b * pos_sb + t * pos_ss]);
  for (int e = threadIdx.x; e < H * per_head; e += blockDim.x) {
    const int h = e / per_head, i = (e - h * per_head) * VEC;
    T* p = q + (row * H + h) * (dim + rot) + dim + i;
    float u[VEC], v[VEC];
    load_vec<T, VEC>(p, u);
    load_vec<T, VEC>(p + half, v);
#pragma unroll
    for (int j = 0; j < VEC; ++j) turn(at * freq[i + j], u[j], v[j]);
    store_vec<T, VEC>(p, u);
    store_vec<T, VEC>(p + half, v);
  }
}

// what a decode step's query carries besides the part that meets W_uk
struct QueryTail {
  int rot;                             // 0: nothing
  const long long* pos; long long pos_sb;
  const float* freq;
};
// columns R .. R + rot of qa for rows b0 .. b0 + nb, head h: the query's rotated part, scaled
template <typename T>
__device__ __forceinline__ void absorb_tail(const T* q, long long ldq, float* qa, const QueryTail& x, int b0, int nb, int h, int H,
                                            int dim, int R, float scale) {
  const int half = x.rot / 2;
  for (int e = threadIdx.x; e < nb * half; e += blockDim.x) {
    const int b = b0 + e / half, i = e % half;
    const T* src = q + b * ldq + static_cast<long long>(h) * (dim + x.rot) + dim + i;
    float u = Num<T>::to(src[0]), v = Num<T>::to(src[half]);
    turn(static_cast<float>(x.pos[b * x.pos_sb]) * x.freq[i], u, v);
    float* dst = qa + (static_cast<long long>(b) * H + h) * (R + x.rot) + R + i;
    dst[0] = u * scale;
    dst[half] = v * scale;
  }
}

// qa[b, h, r] = scale * sum_d q[b, h * dim + d] * w_uk[h * dim + d, r]; block = (64 columns r, head, NB rows b)
template <typename T, int VEC, int NB>
__global__ void __launch_bounds__(256) latent_absorb_kernel(const T* __restrict__ q, long long ldq, const T* __restrict__ w,
                                                            long long ldw, float* __restrict__ qa, int B, int H, int dim,
                                                            int R, float scale, const QueryTail tail) {
  constexpr int CW = 64, CP = CW / VEC, DG = 256 / CP;   // VEC columns per thread, DG groups of rows d
  extern __shared__ float ab_smem[];
  float* qs = ab_smem;                 // [NB][dim]
  float* part = qs + NB * dim;         // [DG][CW], one row b at a time
  const int h = blockIdx.y, r0 = blockIdx.x * CW, b0 = blockIdx.z * NB;
  const int nb = min(NB, B - b0);
  if (r0 >= R) {                       // one more block along the columns when there is a rotated part
    absorb_tail<T>(q, ldq, qa, tail, b0, nb, h, H, dim, R, scale);
    return;
  }
  for (int b = 0; b < nb; ++b)
    for (int d = threadIdx.x; d < dim; d += 256)
      qs[b * dim + d] = Num<T>::to(q[(b0 + b) * ldq + static_cast<long long>(h) * (dim + tail.rot) + d]) * scale;
  __syncthreads();
  const int cp = threadIdx.x % CP, dg = threadIdx.x / CP;
  const int r = r0 + cp * VEC;
  float acc[NB][VEC];
#pragma unroll
  for (int b = 0; b < NB; ++b)
#pragma unroll
    for (int i = 0; i < VEC; ++i) acc[b][i] = 0.f;
  if (r < R) {                         // VEC > 1: the launcher guarantees R % VEC == 0
    const T* wr = w + static_cast<long long>(h) * dim * ldw + r;
#pragma unroll 4
    for (int d = dg; d < dim; d += DG) {
      float v[VEC];
      load_vec<T, VEC>(wr + d * ldw, v);
#pragma unroll
      for (int b = 0; b < NB; ++b) {
        const float x = b < nb ? qs[b * dim + d] : 0.f;
#pragma unroll
        for (int i = 0; i < VEC; ++i) acc[b][i] = fmaf(x, v[i], acc[b][i]);
      }
    }
  }
#pragma unroll
  for (int b = 0; b < NB; ++b) {
    if (b >= nb) break;                // uniform over the block
    __syncthreads();
#pragma unroll
    for (int i = 0; i < VEC; ++i) part[dg * CW + cp * VEC + i] = acc[b][i];
    __syncthreads();
    if (threadIdx.x < CW && r0 + threadIdx.x < R) {
      float t = 0.f;
#pragma unroll
      for (int g = 0; g < DG; ++g) t += part[g * CW + threadIdx.x];
      qa[(static_cast<long long>(b0 + b) * H + h) * (R + tail.rot) + r0 + threadIdx.x] = t;
    }
  }
}

struct LatentDecodeParams {
  const float* qa;                     // [B, H, W], scaled
  const void* cache;                   // [B, Tmax, W]
  const int* lengths;                  // [B] valid positions
  const uint8_t* keep; long long ld_keep; int n_keep;   // [B, n_keep], 0 = padded, or nullptr
  float* ws;                           // [B, H, splits, ldw]: sum p c; ldw = R rounded up to a multiple of 4
  float* stat;                         // [B, H, splits, 2]: max, sum p
  int B, H, R, W, ldw, Tmax, splits;   // W = R + rotated part: the width of the scores' vectors
  int gate_wide;                       // the output gate has a column per output column
  int* err;
};

constexpr int LD_HEADS = 16, LD_KEYS = 16;

// scalar version: any R, any type; block = (slice, head group, row)
template <typename T, int NR>
__global__ void __launch_bounds__(256) latent_decode_kernel(const LatentDecodeParams p) {
  extern __shared__ float ld_smem[];
  const int rp = p.W + 1;
  float* qs = ld_smem;                 // [LD_HEADS][W + 1]
  float* cs = qs + LD_HEADS * rp;      // [LD_KEYS][W + 1]
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
  for (int e = tid; e < nh * p.W; e += 256)
    qs[(e / p.W) * rp + e % p.W] = p.qa[(static_cast<long long>(b) * p.H + h0) * p.W + e];
  for (int e = tid; e < (LD_HEADS - nh) * p.W; e += 256) qs[(nh + e / p.W) * rp + e % p.W] = 0.f;
  if (tid < LD_HEADS) { ms[tid] = -CUDART_INF_F; ls[tid] = 0.f; }
  float acc[NR][LD_HEADS];
#pragma unroll
  for (int j = 0; j < NR; ++j)
#pragma unroll
    for (int a = 0; a < LD_HEADS; ++a) acc[j][a] = 0.f;
  const T* c = static_cast<const T*>(p.cache) + static_cast<long long>(b) * p.Tmax * p.W;
  for (int k0 = t0; k0 < t1; k0 += LD_KEYS) {
    const int n = min(LD_KEYS, t1 - k0);
    __syncthreads();
    for (int e = tid; e < LD_KEYS * p.W; e += 256) {
      const int t = e / p.W, r = e % p.W;
      cs[t * rp + r] = t < n ? Num<T>::to(c[static_cast<long long>(k0 + t) * p.W + r]) : 0.f;
    }
    __syncthreads();
    {
      const int a = tid >> 4, t = tid & 15;
      float d = 0.f;
      for (int r = 0; r < p.W; ++r) d = fmaf(qs[a * rp + r], cs[t * rp + r], d);
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
    const long long at = (static_cast<long long>(b) * p.H + h0 + a) * p.splits + sp;
    float* w = p.ws + at * p.ldw;
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
    if (tid == 0) { p.stat[at * 2] = ms[a]; p.stat[at * 2 + 1] = ls[a]; }
  }
}

// 16-bit version on the tensor cores for R % 16 == 0 and W % 16 == 0: MT x 16 heads are the rows of m16n8k16 tiles, so the cache streams
// through shared memory once for all of them. 8 warps, LM_KT cached vectors per step:
//   scores  warp = (16 heads) x (16 of the keys) x (a half or a quarter of W); q' as 16-bit, 32-bit sums
//   softmax warp w owns heads 2 MT w ..; lane = key; running max and sum in registers, P is stored as 16-bit
//   output  a warp owns every eighth pair of 8-column blocks of R; the cached vectors are read transposed
// The next vectors are fetched with cp.async meanwhile, and two blocks per SM overlap each other's phases.
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
__device__ __forceinline__ void ldsm2_t(uint32_t addr, uint32_t& r0, uint32_t& r1) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void ldsm4_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}

// 16-bit, 16 rows b at a time on the tensor cores: qa[b, h, r] = scale * sum_d q[b, d] w_uk[d, r]. Block = (64 columns r, head,
// 16 rows); W_uk's [dim, 64] tile goes through shared memory and is read transposed; dim % 16 == 0, R % 8 == 0.
template <typename T>
__global__ void __launch_bounds__(256) latent_absorb_mma_kernel(const T* __restrict__ q, long long ldq, const T* __restrict__ w,
                                                                long long ldw, float* __restrict__ qa, int B, int H, int dim,
                                                                int R, float scale, const QueryTail tail) {
  constexpr int CW = 64, WP = CW + 8;
  extern __shared__ __align__(16) uint8_t am_smem[];
  const int qp = dim + 8;
  T* qs = reinterpret_cast<T*>(am_smem);   // [16][qp]
  T* wsm = qs + 16 * qp;                   // [dim][WP]
  const int h = blockIdx.y, r0 = blockIdx.x * CW, b0 = blockIdx.z * 16;
  const int nb = min(16, B - b0), nc = min(CW, R - r0) / 8;   // 16-byte pieces of a tile row
  if (r0 >= R) {                           // one more block along the columns when there is a rotated part
    absorb_tail<T>(q, ldq, qa, tail, b0, nb, h, H, dim, R, scale);
    return;
  }
  for (int e = threadIdx.x; e < dim * 8; e += 256) {
    const int d = e >> 3, v = e & 7;
    const bool in = v < nc;                // columns past R are zero-filled
    const T* src = w + (static_cast<long long>(h) * dim + d) * ldw + r0 + (in ? v * 8 : 0);
    const int bytes = in ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(wsm + d * WP + v * 8)), "l"(src), "r"(bytes) : "memory");
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  for (int e = threadIdx.x; e < 16 * dim; e += 256) {
    const int b = e / dim, d = e - b * dim;
    qs[b * qp + d] = b < nb ? q[(b0 + b) * ldq + static_cast<long long>(h) * (dim + tail.rot) + d] : Num<T>::from(0.f);
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
  for (int s = 0; s < dim / 16; ++s) {
    uint32_t a[4], b0r, b1r;
    ldsm4(smem_u32(qs + (lane & 15) * qp + s * 16 + (lane >> 4) * 8), a);
    ldsm2_t(smem_u32(wsm + (s * 16 + (lane & 15)) * WP + warp * 8), b0r, b1r);
    MmaT<T>::mma(acc, a, b0r, b1r);
  }
  const int col = r0 + warp * 8 + (lane & 3) * 2;
  if (col < R) {                           // R is even
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int b = (lane >> 2) + 8 * hf;
      if (b < nb)
        *reinterpret_cast<float2*>(qa + (static_cast<long long>(b0 + b) * H + h) * (R + tail.rot) + col) =
            make_float2(acc[hf * 2] * scale, acc[hf * 2 + 1] * scale);
    }
  }
}

constexpr int LM_KT = 32;

template <typename T, int MT, int NP>   // MT groups of 16 heads, NP pairs of 8-column blocks per warp
__global__ void __launch_bounds__(256, NP <= 4 ? 2 : 1) latent_decode_mma_kernel(const LatentDecodeParams p) {
  constexpr int HM = 16 * MT, PP = LM_KT + 8, SP = LM_KT + 1, KS = 4 / MT;
  extern __shared__ __align__(16) uint8_t lm_smem[];
  const int rp = p.W + 8;               // padded row: 16-byte aligned, conflict-free ldmatrix
  T* qs = reinterpret_cast<T*>(lm_smem);            // [HM][rp]
  T* cs = qs + HM * rp;                             // [2][LM_KT][rp]
  T* ps = cs + 2 * LM_KT * rp;                      // [HM][PP]
  float* ss = reinterpret_cast<float*>(ps + HM * PP);   // [KS][HM][SP]
  float* fac = ss + KS * HM * SP;                // [HM]
  const int b = blockIdx.z, h0 = blockIdx.y * HM, sp = blockIdx.x, tid = threadIdx.x;
  const int warp = tid >> 5, lane = tid & 31;
  const int nh = min(HM, p.H - h0);
  int len = p.lengths[b];
  if (len < 0 || len > p.Tmax) {       // a length that does not fit the cache: never read past it
    if (tid == 0) OSLO_REPORT_BOUNDS(p.err);
    len = len < 0 ? 0 : p.Tmax;
  }
  const int tiles = (len + LM_KT - 1) / LM_KT, per = (tiles + p.splits - 1) / p.splits * LM_KT;
  const int t0 = sp * per, t1 = min(len, t0 + per);
  const T* c = static_cast<const T*>(p.cache) + static_cast<long long>(b) * p.Tmax * p.W;
  const int vr = p.W / 8;              // 16-byte pieces of a cached vector
  const int dt = 256 / vr, dv = 256 % vr, ft = tid / vr, fv = tid % vr;
  auto fetch = [&](int k0, int buf) {
    T* dst = cs + static_cast<size_t>(buf) * LM_KT * rp;
    int t = ft, v = fv;
    while (t < LM_KT) {
      const uint32_t d32 = smem_u32(dst + t * rp + v * 8);
      const bool in = k0 + t < t1;     // rows past the slice are zero-filled (source size 0)
      const T* src = c + static_cast<long long>(in ? k0 + t : 0) * p.W + v * 8;
      const int bytes = in ? 16 : 0;
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d32), "l"(src), "r"(bytes) : "memory");
      t += dt;
      v += dv;
      if (v >= vr) { v -= vr; ++t; }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (t0 < t1) fetch(t0, 0);
  for (int a = warp; a < HM; a += 8) {
    const float* src = p.qa + (static_cast<long long>(b) * p.H + h0 + a) * p.W;
#pragma unroll 4
    for (int r = lane * 4; r < p.W; r += 128) {
      float x[4] = {0.f, 0.f, 0.f, 0.f};
      if (a < nh) load_vec<float, 4>(src + r, x);
      store_vec<T, 4>(qs + a * rp + r, x);
    }
  }
  float acc[MT][NP][2][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int j = 0; j < NP; ++j)
#pragma unroll
      for (int u = 0; u < 2; ++u)
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[m][j][u][i] = 0.f;
  float m_run[2 * MT], l_run[2 * MT];
#pragma unroll
  for (int u = 0; u < 2 * MT; ++u) { m_run[u] = -CUDART_INF_F; l_run[u] = 0.f; }
  const int arow = lane & 15, acol = (lane >> 4) * 8;      // ldmatrix.x4 source of an A fragment
  const int kg = warp & 1, mt = (warp >> 1) % MT, ks = (warp >> 1) / MT;
  const int n16 = p.W / 16, s_begin = ks * n16 / KS, s_end = (ks + 1) * n16 / KS;
  // B fragments of 16 keys x 16 columns: matrices (keys 0-7, cols 0-7), (keys 0-7, cols 8-15), (keys 8-15, ...)
  const int brow = kg * 16 + (lane & 7) + ((lane >> 4) << 3), bcol = ((lane >> 3) & 1) * 8;
  for (int k0 = t0, it = 0; k0 < t1; k0 += LM_KT, ++it) {
    const int buf = it & 1;
    if (k0 + LM_KT < t1) {                                 // the other buffer was last read before the closing barrier
      fetch(k0 + LM_KT, buf ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const T* ct = cs + static_cast<size_t>(buf) * LM_KT * rp;
    {
      float d[2][4];
#pragma unroll
      for (int u = 0; u < 2; ++u)
#pragma unroll
        for (int i = 0; i < 4; ++i) d[u][i] = 0.f;
#pragma unroll 4
      for (int s = s_begin; s < s_end; ++s) {
        uint32_t a[4], bb[4];
        ldsm4(smem_u32(ct + brow * rp + s * 16 + bcol), bb);
        ldsm4(smem_u32(qs + (mt * 16 + arow) * rp + s * 16 + acol), a);
        MmaT<T>::mma(d[0], a, bb[0], bb[1]);
        MmaT<T>::mma(d[1], a, bb[2], bb[3]);
      }
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        float* o = ss + (ks * HM + mt * 16 + (lane >> 2)) * SP + kg * 16 + u * 8 + (lane & 3) * 2;
        o[0] = d[u][0]; o[1] = d[u][1];
        o[8 * SP] = d[u][2]; o[8 * SP + 1] = d[u][3];
      }
    }
    __syncthreads();
    {
      const int pos = k0 + lane;
      const bool vis = pos < t1 && (p.keep == nullptr || pos >= p.n_keep || p.keep[b * p.ld_keep + pos]);
      float x[2 * MT], mx[2 * MT], sum[2 * MT];
#pragma unroll
      for (int u = 0; u < 2 * MT; ++u) {
        const float* o = ss + (warp * 2 * MT + u) * SP + lane;
        float v = o[0];
#pragma unroll
        for (int k = 1; k < KS; ++k) v += o[k * HM * SP];
        x[u] = vis ? v : -CUDART_INF_F;
        mx[u] = fmaxf(m_run[u], x[u]);
      }
#pragma unroll
      for (int off = 16; off > 0; off >>= 1)
#pragma unroll
        for (int u = 0; u < 2 * MT; ++u) mx[u] = fmaxf(mx[u], __shfl_xor_sync(0xffffffffu, mx[u], off));
#pragma unroll
      for (int u = 0; u < 2 * MT; ++u) {
        sum[u] = x[u] == -CUDART_INF_F ? 0.f : expf(x[u] - mx[u]);
        ps[(warp * 2 * MT + u) * PP + lane] = Num<T>::from(sum[u]);
      }
#pragma unroll
      for (int off = 16; off > 0; off >>= 1)
#pragma unroll
        for (int u = 0; u < 2 * MT; ++u) sum[u] += __shfl_xor_sync(0xffffffffu, sum[u], off);
#pragma unroll
      for (int u = 0; u < 2 * MT; ++u) {
        const float f = m_run[u] == -CUDART_INF_F ? 0.f : expf(m_run[u] - mx[u]);
        l_run[u] = l_run[u] * f + sum[u];
        m_run[u] = mx[u];
        if (lane == 0) fac[warp * 2 * MT + u] = f;
      }
    }
    __syncthreads();
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float f0 = fac[m * 16 + (lane >> 2)], f1 = fac[m * 16 + (lane >> 2) + 8];
#pragma unroll
      for (int j = 0; j < NP; ++j)
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          acc[m][j][u][0] *= f0; acc[m][j][u][1] *= f0; acc[m][j][u][2] *= f1; acc[m][j][u][3] *= f1;
        }
    }
#pragma unroll
    for (int s = 0; s < LM_KT / 16; ++s) {
      uint32_t a[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) ldsm4(smem_u32(ps + (m * 16 + arow) * PP + s * 16 + acol), a[m]);
#pragma unroll
      for (int j = 0; j < NP; ++j) {
        const int col = (warp + 8 * j) * 16;
        if (col < p.R) {                                   // uniform over the warp
          uint32_t bb[4];
          ldsm4_t(smem_u32(ct + (s * 16 + (lane & 15)) * rp + col + (lane >> 4) * 8), bb);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            MmaT<T>::mma(acc[m][j][0], a[m], bb[0], bb[1]);
            MmaT<T>::mma(acc[m][j][1], a[m], bb[2], bb[3]);
          }
        }
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int j = 0; j < NP; ++j) {
      const int col = (warp + 8 * j) * 16;
      if (col >= p.R) continue;
#pragma unroll
      for (int u = 0; u < 2; ++u)
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
          const int a = m * 16 + (lane >> 2) + 8 * hf;
          if (a < nh) {
            float* w = p.ws + ((static_cast<long long>(b) * p.H + h0 + a) * p.splits + sp) * p.ldw + col + u * 8 + (lane & 3) * 2;
            *reinterpret_cast<float2*>(w) = make_float2(acc[m][j][u][hf * 2], acc[m][j][u][hf * 2 + 1]);
          }
        }
    }
#pragma unroll
  for (int u = 0; u < 2 * MT; ++u) {
    const int a = warp * 2 * MT + u;
    if (lane == 0 && a < nh) {
      float* w = p.stat + ((static_cast<long long>(b) * p.H + h0 + a) * p.splits + sp) * 2;
      w[0] = m_run[u];
      w[1] = l_run[u];
    }
  }
}
static size_t latent_mma_smem(int W, int mt) {
  const size_t rp = W + 8, hm = 16 * mt;
  return (hm * rp + 2 * LM_KT * rp + hm * (LM_KT + 8)) * 2 + (4 / mt * hm * (LM_KT + 1) + hm) * sizeof(float);
}

// the slice weights of one row (all lanes of a warp): wt[s] = exp(max_s - max) * gate / denominator; sink -inf: none
template <typename T>
__device__ __forceinline__ void slice_weights(const LatentDecodeParams& p, int b, int h, float snk, float gate, float* wt, int lane) {
  const float2* st = reinterpret_cast<const float2*>(p.stat) + (static_cast<long long>(b) * p.H + h) * p.splits;
  float m = snk;
  for (int s = lane; s < p.splits; s += 32) m = fmaxf(m, st[s].x);
#pragma unroll
  for (int off = 16; off > 0; off >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, off));
  if (m == -CUDART_INF_F) m = 0.f;     // no visible key: all terms are zero
  float tot = 0.f;
  for (int s = lane; s < p.splits; s += 32) {
    const float2 ml = st[s];
    const float f = ml.x == -CUDART_INF_F ? 0.f : expf(ml.x - m);
    tot += f * ml.y;
    wt[s] = f;
  }
  const float den = warp_sum(tot) + expf(snk - m);
  const float g = den > 0.f ? gate / den : 0.f;
  for (int s = lane; s < p.splits; s += 32) wt[s] *= g;
}

// out[b, h * vdim + j] = sigmoid(g) * sum_r w_uv[h * vdim + j, r] * o[r],  o = merged slices / (sum + exp(sink))
// for NB rows b per block, so that W_uv is read once for all of them; a warp computes 4 of the j at a time
template <typename T, int VEC, int NB>
__global__ void __launch_bounds__(256) latent_finish_kernel(const LatentDecodeParams p, const T* __restrict__ w, long long ldw,
                                                            const T* __restrict__ sink, const T* __restrict__ gate,
                                                            long long ldg, T* __restrict__ out, int vdim, int rows_per_block) {
  extern __shared__ __align__(16) float fin_smem[];   // [NB][p.ldw] then [NB][splits] weights
  float* o = fin_smem;
  float* wt = fin_smem + NB * p.ldw;
  const int h = blockIdx.y, b0 = blockIdx.z * NB, nb = min(NB, p.B - b0), R = p.R, splits = p.splits;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const float snk = sink ? Num<T>::to(sink[h]) : -CUDART_INF_F;
  for (int i = warp; i < nb; i += 8)
    slice_weights<T>(p, b0 + i, h, snk, p.gate_wide ? 1.f : sigmoid_f(Num<T>::to(gate[(b0 + i) * ldg + h])), wt + i * splits, lane);
  __syncthreads();
  const int quads = p.ldw / 4;
  for (int e = threadIdx.x; e < nb * quads; e += 256) {
    const int i = e / quads, c = e - i * quads;
    const float* base = p.ws + (static_cast<long long>(b0 + i) * p.H + h) * splits * p.ldw + c * 4;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int s = 0; s < splits; ++s) {
      const float4 x = *reinterpret_cast<const float4*>(base + static_cast<long long>(s) * p.ldw);
      const float f = wt[i * splits + s];
      v.x = fmaf(f, x.x, v.x); v.y = fmaf(f, x.y, v.y); v.z = fmaf(f, x.z, v.z); v.w = fmaf(f, x.w, v.w);
    }
    *reinterpret_cast<float4*>(o + i * p.ldw + c * 4) = v;   // columns past R are never read below
  }
  __syncthreads();
  constexpr int JR = 4;
  const int j1 = min(vdim, (static_cast<int>(blockIdx.x) + 1) * rows_per_block);
  for (int j = blockIdx.x * rows_per_block + warp * JR; j < j1; j += 8 * JR) {
    const T* wr = w + (static_cast<long long>(h) * vdim + j) * ldw;
    const int nj = min(JR, j1 - j);
    float acc[JR][NB];
#pragma unroll
    for (int a = 0; a < JR; ++a)
#pragma unroll
      for (int i = 0; i < NB; ++i) acc[a][i] = 0.f;
#pragma unroll 2
    for (int k = lane * VEC; k < R; k += 32 * VEC) {
      float x[JR][VEC];
#pragma unroll
      for (int a = 0; a < JR; ++a)
        if (a < nj) load_vec<T, VEC>(wr + a * ldw + k, x[a]);
        else {
#pragma unroll
          for (int u = 0; u < VEC; ++u) x[a][u] = 0.f;
        }
#pragma unroll
      for (int i = 0; i < NB; ++i)
        if (i < nb) {
#pragma unroll
          for (int u = 0; u < VEC; ++u) {
            const float y = o[i * p.ldw + k + u];
#pragma unroll
            for (int a = 0; a < JR; ++a) acc[a][i] = fmaf(x[a][u], y, acc[a][i]);
          }
        }
    }
#pragma unroll
    for (int a = 0; a < JR; ++a)
#pragma unroll
      for (int i = 0; i < NB; ++i) {
        const float d = warp_sum(acc[a][i]);
        if (lane == 0 && i < nb && a < nj) {
          const float g = p.gate_wide ? sigmoid_f(Num<T>::to(gate[(b0 + i) * ldg + static_cast<long long>(h) * vdim + j + a])) : 1.f;
          out[(static_cast<long long>(b0 + i) * p.H + h) * vdim + j + a] = Num<T>::from(d * g);
        }
      }
  }
}

// 16-bit, 16 rows b at a time on the tensor cores; R % 32 == 0, vdim % 8 == 0. A lane fetches 8 consecutive elements of its
// column's W_uv row with one load and uses them as two k steps; the A operand is permuted alike, so no shuffles are needed.
template <typename T>
__global__ void __launch_bounds__(256) latent_finish_mma_kernel(const LatentDecodeParams p, const T* __restrict__ w, long long ldw,
                                                                const T* __restrict__ sink, const T* __restrict__ gate,
                                                                long long ldg, T* __restrict__ out, int vdim) {
  extern __shared__ __align__(16) uint8_t fm_smem[];
  const int op = p.R + 8, quads = p.R / 4;
  T* o = reinterpret_cast<T*>(fm_smem);                    // [16][op]
  float* wt = reinterpret_cast<float*>(o + 16 * op);       // [16][splits]
  const int h = blockIdx.y, b0 = blockIdx.z * 16, nb = min(16, p.B - b0);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const float snk = sink ? Num<T>::to(sink[h]) : -CUDART_INF_F;
  for (int i = warp; i < nb; i += 8)
    slice_weights<T>(p, b0 + i, h, snk, p.gate_wide ? 1.f : sigmoid_f(Num<T>::to(gate[(b0 + i) * ldg + h])), wt + i * p.splits, lane);
  __syncthreads();
#pragma unroll 2
  for (int e = threadIdx.x; e < 16 * quads; e += 256) {
    const int i = e / quads, c = e - i * quads;
    float v[4] = {0.f, 0.f, 0.f, 0.f};
    if (i < nb) {
      const float* base = p.ws + (static_cast<long long>(b0 + i) * p.H + h) * p.splits * p.ldw + c * 4;
#pragma unroll 4
      for (int s = 0; s < p.splits; ++s) {
        const float4 x = *reinterpret_cast<const float4*>(base + static_cast<long long>(s) * p.ldw);
        const float f = wt[i * p.splits + s];
        v[0] = fmaf(f, x.x, v[0]); v[1] = fmaf(f, x.y, v[1]); v[2] = fmaf(f, x.z, v[2]); v[3] = fmaf(f, x.w, v[3]);
      }
    }
    store_vec<T, 4>(o + i * op + c * 4, v);
  }
  __syncthreads();
  const int g = lane >> 2, t = lane & 3;
  for (int j0 = (blockIdx.x * 8 + warp) * 8; j0 < vdim; j0 += gridDim.x * 64) {
    const T* wr = w + (static_cast<long long>(h) * vdim + j0 + g) * ldw + t * 8;
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 8
    for (int k = 0; k < p.R; k += 32) {
      const uint4 bv = *reinterpret_cast<const uint4*>(wr + k);
      const uint4 a0 = *reinterpret_cast<const uint4*>(o + g * op + k + t * 8);
      const uint4 a1 = *reinterpret_cast<const uint4*>(o + (g + 8) * op + k + t * 8);
      const uint32_t s0[4] = {a0.x, a1.x, a0.y, a1.y}, s1[4] = {a0.z, a1.z, a0.w, a1.w};
      MmaT<T>::mma(acc, s0, bv.x, bv.y);
      MmaT<T>::mma(acc, s1, bv.z, bv.w);
    }
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int b = g + 8 * hf;
      if (b < nb) {
        float v[2] = {acc[hf * 2], acc[hf * 2 + 1]};
        if (p.gate_wide) {                 // the gate's rows need not be aligned
          const T* g = gate + (b0 + b) * ldg + static_cast<long long>(h) * vdim + j0 + t * 2;
          v[0] *= sigmoid_f(Num<T>::to(g[0]));
          v[1] *= sigmoid_f(Num<T>::to(g[1]));
        }
        store_vec<T, 2>(out + (static_cast<long long>(b0 + b) * p.H + h) * vdim + j0 + t * 2, v);
      }
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
                                   long long ldg, void* out, int B, int H, int G, int KG, int Sq, int Sk, int dim, int vdim, float scale,
                                   float softcap, int window, int keep_first, const int* lead, int gate_wide, int dtype,
                                   cudaStream_t stream) {
  using namespace oslo;
  if (B <= 0 || H <= 0 || Sq <= 0) return 0;
  if (Sk < Sq || B > 65535 || H > 65535 || G <= 0 || H % G || KG <= 0 || H % KG) return -1;
  SinkAttnParams p{q, k, v, q_sb, q_ss, q_sh, k_sb, k_ss, k_sh, v_sb, v_ss, v_sh, keep, ld_keep, sink, gate, ldg, out,
                   B, H, G, KG, Sq, Sk, dim, vdim, scale, softcap, window, keep_first, lead, gate_wide};
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
                                float eps, int B, int S, int rot, const long long* pos, long long pos_sb, long long pos_ss,
                                const float* freq, void* c_out, int dtype, int* err_word, cudaStream_t stream) {
  using namespace oslo;
  if (B <= 0 || S <= 0) return 0;
  const long long rows = static_cast<long long>(B) * S;
  if (rows > 0x7fffffffll || rot < 0 || rot % 2 || (rot > 0 && (pos == nullptr || freq == nullptr))) return -1;
  const LatentPrepParams p{cq, wq, ldq, q_rank, cq_out, ckv, wkv, ldkv, kv_rank, rot, cache, c_out, lengths, pos, pos_sb, pos_ss,
                           freq, S, Tmax, eps, err_word};
  const size_t a4 = dtype == OSLO_DT_FP32 ? 16 : 8;
  bool vec = q_rank % 4 == 0 && kv_rank % 4 == 0 && rot % 4 == 0 && ldq % 4 == 0 && ldkv % 4 == 0;
  for (const void* t : {cq, wq, static_cast<const void*>(cq_out), ckv, wkv, static_cast<const void*>(cache), static_cast<const void*>(c_out)})
    vec = vec && aligned_to(t, a4);        // null is aligned
  const int widest = std::max(q_rank, kv_rank) / (vec ? 4 : 1), threads = widest <= 64 ? 64 : (widest <= 128 ? 128 : 256);
  const dim3 grid(static_cast<unsigned>(rows), ckv ? 2 : 1);
  OSLO_DISPATCH_T(dtype, {
    if (vec) latent_prep_kernel<T, 4><<<grid, threads, 0, stream>>>(p);
    else latent_prep_kernel<T, 1><<<grid, threads, 0, stream>>>(p);
  });
  return static_cast<int>(cudaGetLastError());
}

extern "C" int oslo_rotate_halves(void* q, const long long* pos, long long pos_sb, long long pos_ss, const float* freq, int B, int S,
                                  int H, int dim, int rot, int dtype, cudaStream_t stream) {
  using namespace oslo;
  const long long rows = static_cast<long long>(B) * S;
  if (rows <= 0 || H <= 0 || rot <= 0) return 0;
  if (rows > 0x7fffffffll || rot % 2) return -1;
  const size_t a4 = dtype == OSLO_DT_FP32 ? 16 : 8;
  const bool vec = rot % 8 == 0 && dim % 4 == 0 && aligned_to(q, a4);
  const int per_head = rot / 2 / (vec ? 4 : 1);
  const unsigned grid = static_cast<unsigned>(rows), threads = std::min(256, (H * per_head + 31) / 32 * 32);
  OSLO_DISPATCH_T(dtype, {
    if (vec) rotate_halves_kernel<T, 4><<<grid, threads, 0, stream>>>(static_cast<T*>(q), pos, pos_sb, pos_ss, freq, S, H, dim, rot, per_head);
    else rotate_halves_kernel<T, 1><<<grid, threads, 0, stream>>>(static_cast<T*>(q), pos, pos_sb, pos_ss, freq, S, H, dim, rot, per_head);
  });
  return static_cast<int>(cudaGetLastError());
}

namespace oslo {

template <typename T>
static int latent_scan(const LatentDecodeParams& p, int use_mma, cudaStream_t st) {
  if constexpr (sizeof(T) == 2) {
    if (use_mma) {
      const int mt = p.H > LD_HEADS ? 2 : 1, np = (p.R + 127) / 128;
      const size_t smem = latent_mma_smem(p.W, mt);
      dim3 grid(p.splits, (p.H + 16 * mt - 1) / (16 * mt), p.B);
#define LM_GO(MT, NP)                                                                                   \
  {                                                                                                     \
    const int rc = set_smem(reinterpret_cast<const void*>(&latent_decode_mma_kernel<T, MT, NP>), smem); \
    if (rc) return rc;                                                                                  \
    latent_decode_mma_kernel<T, MT, NP><<<grid, 256, smem, st>>>(p);                                    \
    return static_cast<int>(cudaGetLastError());                                                        \
  }
      if (mt == 1) {
        if (np == 1) LM_GO(1, 1)
        if (np == 2) LM_GO(1, 2)
        if (np <= 4) LM_GO(1, 4)
        LM_GO(1, 8)
      }
      if (np == 1) LM_GO(2, 1)
      if (np == 2) LM_GO(2, 2)
      if (np <= 4) LM_GO(2, 4)
      LM_GO(2, 8)
#undef LM_GO
    }
  }
  dim3 grid(p.splits, (p.H + LD_HEADS - 1) / LD_HEADS, p.B);
  const size_t smem = (static_cast<size_t>(LD_HEADS + LD_KEYS) * (p.W + 1) + LD_HEADS * LD_KEYS) * sizeof(float);
#define LD_GO(NR)                                                                               \
  {                                                                                             \
    const int rc = set_smem(reinterpret_cast<const void*>(&latent_decode_kernel<T, NR>), smem); \
    if (rc) return rc;                                                                          \
    latent_decode_kernel<T, NR><<<grid, 256, smem, st>>>(p);                                    \
  }
  if (p.R <= 256) LD_GO(1)
  else if (p.R <= 512) LD_GO(2)
  else LD_GO(4)
#undef LD_GO
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int VEC>
static int latent_absorb(const LatentDecodeParams& p, const void* q, long long ldq, const void* w, long long ldw, float* qa,
                         int dim, float scale, const QueryTail& tail, cudaStream_t st) {
  const int extra = tail.rot > 0 ? 1 : 0;  // a block of its own for the rotated part
  if constexpr (sizeof(T) == 2 && VEC == 8) {
    if (p.B > 2 && dim % 16 == 0) {
      const size_t smem = (16 * static_cast<size_t>(dim + 8) + static_cast<size_t>(dim) * 72) * 2;
      const int rc = set_smem(reinterpret_cast<const void*>(&latent_absorb_mma_kernel<T>), smem);
      if (rc) return rc;
      latent_absorb_mma_kernel<T><<<dim3((p.R + 63) / 64 + extra, p.H, (p.B + 15) / 16), 256, smem, st>>>(
          static_cast<const T*>(q), ldq, static_cast<const T*>(w), ldw, qa, p.B, p.H, dim, p.R, scale, tail);
      return static_cast<int>(cudaGetLastError());
    }
  }
  const int nb = p.B >= 8 ? 8 : (p.B >= 2 ? 2 : 1);
  const size_t smem = (static_cast<size_t>(nb) * dim + 256 * VEC) * sizeof(float);
  dim3 grid((p.R + 63) / 64 + extra, p.H, (p.B + nb - 1) / nb);
#define AB_GO(NB)                                                                                                       \
  {                                                                                                                     \
    const int rc = set_smem(reinterpret_cast<const void*>(&latent_absorb_kernel<T, VEC, NB>), smem);                    \
    if (rc) return rc;                                                                                                  \
    latent_absorb_kernel<T, VEC, NB><<<grid, 256, smem, st>>>(static_cast<const T*>(q), ldq, static_cast<const T*>(w), ldw, qa, \
                                                              p.B, p.H, dim, p.R, scale, tail);                         \
  }
  if (nb == 8) AB_GO(8)
  else if (nb == 2) AB_GO(2)
  else AB_GO(1)
#undef AB_GO
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int VEC>
static int latent_finish(const LatentDecodeParams& p, const void* w_uv, long long ldv, const void* sink, const void* gate,
                         long long ldg, void* out, int vdim, int num_sms, cudaStream_t st) {
  if constexpr (sizeof(T) == 2 && VEC == 8) {
    if (p.B > 2 && p.R % 32 == 0 && vdim % 8 == 0) {
      const size_t smem = 16 * (static_cast<size_t>(p.R + 8) * 2 + p.splits * sizeof(float));
      const int rc = set_smem(reinterpret_cast<const void*>(&latent_finish_mma_kernel<T>), smem);
      if (rc) return rc;
      const int zb = (p.B + 15) / 16, tiles = (vdim / 8 + 7) / 8;   // one 8-column block per warp while the GPU has room
      const int parts = static_cast<long long>(zb) * p.H * tiles <= 2 * num_sms ? tiles : 1;
      latent_finish_mma_kernel<T><<<dim3(parts, p.H, zb), 256, smem, st>>>(p, static_cast<const T*>(w_uv), ldv,
                                                                           static_cast<const T*>(sink), static_cast<const T*>(gate),
                                                                           ldg, static_cast<T*>(out), vdim);
      return static_cast<int>(cudaGetLastError());
    }
  }
  const int nb = p.B >= 8 ? 8 : (p.B >= 2 ? 2 : 1), zb = (p.B + nb - 1) / nb;
  int parts = 1;                       // value rows of a head over several blocks while the GPU has room
  while (parts < 16 && static_cast<long long>(zb) * p.H * parts < num_sms && vdim / (2 * parts) >= 16) parts *= 2;
  const int rpb = (vdim + parts - 1) / parts;
  const size_t smem = static_cast<size_t>(nb) * (p.ldw + p.splits) * sizeof(float);
  dim3 grid(parts, p.H, zb);
#define FIN_GO(NB)                                                                                                    \
  latent_finish_kernel<T, VEC, NB><<<grid, 256, smem, st>>>(p, static_cast<const T*>(w_uv), ldv, static_cast<const T*>(sink), \
                                                            static_cast<const T*>(gate), ldg, static_cast<T*>(out), vdim, rpb)
  if (nb == 8) FIN_GO(8);
  else if (nb == 2) FIN_GO(2);
  else FIN_GO(1);
#undef FIN_GO
  return static_cast<int>(cudaGetLastError());
}

}  // namespace oslo

// slices of the cache per (row, head group): fewest waves of blocks (two per SM), then the least work per block
extern "C" int oslo_latent_splits(int B, int H, int T, int num_sms) {
  const int per_block = H > oslo::LD_HEADS ? 2 * oslo::LD_HEADS : oslo::LD_HEADS, groups = (H + per_block - 1) / per_block;
  const int tiles = (T + oslo::LM_KT - 1) / oslo::LM_KT;
  int best = 1;
  double best_cost = 1e30;
  for (int s = 1; s <= 64 && s <= tiles; ++s) {
    const long long blocks = static_cast<long long>(B) * groups * s, waves = (blocks + 2 * num_sms - 1) / (2 * num_sms);
    const double cost = static_cast<double>(waves) * ((tiles + s - 1) / s + 2.0) + 0.08 * s;   // set-up and merge of a slice
    if (cost < best_cost) { best_cost = cost; best = s; }
  }
  return best;
}

extern "C" int oslo_latent_decode(const void* q, long long ldq, const void* w_uk, long long ldk, const void* w_uv, long long ldv,
                                  const void* cache, const int* lengths, const uint8_t* keep, long long ld_keep, int n_keep,
                                  const void* sink, const void* gate, long long ldg, float* qa, float* ws, float* stat, void* out,
                                  int B, int H, int dim, int vdim, int R, int rot, const long long* pos, long long pos_sb,
                                  const float* freq, int gate_wide, int Tmax, int splits, float scale, int num_sms, int dtype,
                                  int* err_word, cudaStream_t stream) {
  using namespace oslo;
  if (B <= 0 || H <= 0) return 0;
  if (R <= 0 || R > 1024 || splits < 1 || splits > 64 || B > 65535 || H > 65535) return -1;
  if (rot < 0 || rot % 2 || (rot > 0 && (pos == nullptr || freq == nullptr))) return -1;
  const int W = R + rot;
  LatentDecodeParams p{qa, cache, lengths, keep, ld_keep, n_keep, ws, stat, B, H, R, W, (R + 3) / 4 * 4, Tmax, splits, gate_wide, err_word};
  const QueryTail tail{rot, pos, pos_sb, freq};
  const size_t te = dtype == OSLO_DT_FP32 ? 4 : 2;
  const int v16 = static_cast<int>(16 / te);
  const bool kv = R % v16 == 0 && ldk % v16 == 0 && aligned_to(w_uk, 16);
  const bool vv = R % v16 == 0 && ldv % v16 == 0 && aligned_to(w_uv, 16);
  OSLO_DISPATCH_T(dtype, {
    constexpr int V = 16 / sizeof(T);
    int rc = kv ? latent_absorb<T, V>(p, q, ldq, w_uk, ldk, qa, dim, scale, tail, stream)
                : latent_absorb<T, 1>(p, q, ldq, w_uk, ldk, qa, dim, scale, tail, stream);
    if (rc) return rc;
    rc = latent_scan<T>(p, R % 16 == 0 && W % 16 == 0 && aligned_to(cache, 16), stream);
    if (rc) return rc;
    return vv ? latent_finish<T, V>(p, w_uv, ldv, sink, gate, ldg, out, vdim, num_sms, stream)
              : latent_finish<T, 1>(p, w_uv, ldv, sink, gate, ldg, out, vdim, num_sms, stream);
  });
  return -2;
}
