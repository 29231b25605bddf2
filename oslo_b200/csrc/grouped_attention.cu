// Grouped-query attention with query / key norms, interleaved rotation, capped scores and a sink in the denominator:
// what comes before the scores (qkv_prep_kernel) and decoding with one query per row (grouped_decode_kernel). Prompts run
// on the tcgen05 flash kernel (attention_sm100.cu) or, in 32-bit, on sink_attention_kernel (latent_attention.cu).
//
// Decode: a block scans a slice of one key / value head's cache for (up to GD_HEADS of) the query heads that share it, so
// every cached byte is read once per block; grouped_finish_kernel merges the slices and adds the sink to the denominator.
#include <math_constants.h>

#include <algorithm>

#include "num.cuh"
#include "oslo_kernels.h"
#include "ptx.cuh"

namespace oslo {

// ------------------------------------------------------------------ norms, rotation, cache append
struct PrepParams {
  const void *q, *k, *v; long long ldq, ldk, ldv;     // row b * S + t
  const void *wq, *wk;                                // [dim]
  const long long* pos; long long pos_sb, pos_ss;
  const float* freq; int n_freq;
  void *q_out, *kc, *vc;                              // [B, S, H, dim], [B, G, Tmax, dim], [B, G, Tmax, vdim]
  const int* lengths;
  int S, H, G, dim, vdim, Tmax;
  long long slots;                                    // B * S * (H + 2 G)
  float eps;
  int* err;
};

// one warp per (token, head): H query heads, G key heads, G value heads
template <typename T>
__global__ void __launch_bounds__(256) qkv_prep_kernel(const PrepParams p) {
  const long long slot = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (slot >= p.slots) return;
  const int per = p.H + 2 * p.G;
  const long long row = slot / per;
  int h = static_cast<int>(slot - row * per);
  const long long b = row / p.S, t = row - b * p.S;
  const bool is_q = h < p.H, is_v = h >= p.H + p.G;
  const T* src;
  T* dst;
  if (is_q) {
    src = static_cast<const T*>(p.q) + row * p.ldq + static_cast<long long>(h) * p.dim;
    dst = static_cast<T*>(p.q_out) + (row * p.H + h) * p.dim;
  } else {
    const long long at = p.lengths[b] + t;
    if (at < 0 || at >= p.Tmax) {                      // never write outside the cache
      if (lane == 0) OSLO_REPORT_BOUNDS(p.err);
      return;
    }
    h -= p.H;
    if (is_v) {
      h -= p.G;
      src = static_cast<const T*>(p.v) + row * p.ldv + static_cast<long long>(h) * p.vdim;
      dst = static_cast<T*>(p.vc) + ((b * p.G + h) * p.Tmax + at) * p.vdim;
      for (int c = lane; c < p.vdim; c += 32) dst[c] = src[c];
      return;
    }
    src = static_cast<const T*>(p.k) + row * p.ldk + static_cast<long long>(h) * p.dim;
    dst = static_cast<T*>(p.kc) + ((b * p.G + h) * p.Tmax + at) * p.dim;
  }
  const T* w = static_cast<const T*>(is_q ? p.wq : p.wk);
  float ss = 0.f;
  for (int c = lane; c < p.dim; c += 32) {
    const float x = Num<T>::to(src[c]);
    ss = fmaf(x, x, ss);
  }
  const float r = 1.0f / sqrtf(warp_sum(ss) / p.dim + p.eps);
  const float at = static_cast<float>(p.pos[b * p.pos_sb + t * p.pos_ss]);
  for (int c = 2 * lane; c < p.dim; c += 64) {         // the pair (c, c + 1)
    const bool two = c + 1 < p.dim;
    float x = Num<T>::to(src[c]) * r * Num<T>::to(w[c]);
    float y = two ? Num<T>::to(src[c + 1]) * r * Num<T>::to(w[c + 1]) : 0.f;
    if ((c >> 1) < p.n_freq) {
      float sn, cs;
      sincosf(at * p.freq[c >> 1], &sn, &cs);
      const float u = x * cs - y * sn;
      y = y * cs + x * sn;
      x = u;
    }
    dst[c] = Num<T>::from(x);
    if (two) dst[c + 1] = Num<T>::from(y);
  }
}

// ------------------------------------------------------------------ decode
struct GroupedParams {
  const void* q;                       // [B, H, dim]
  const void *kc, *vc;                 // [B, G, Tmax, dim / vdim]
  const int* lengths;
  const uint8_t* keep; long long ld_keep; int n_keep;   // [B, n_keep], 0 = padded, or nullptr
  float* ws;                           // [B, H, splits, ldw]: sum p v; ldw = vdim rounded up to a multiple of 4
  float* stat;                         // [B, H, splits, 2]: max, sum p
  int H, G, dim, vdim, ldw, Tmax, splits;
  float scale, softcap;
  int* err;
};

constexpr int GD_HEADS = 8, GD_KEYS = 32;

// any head sizes, any type, 32-bit arithmetic; block = (slice, (key head, tile of its query heads), row), NR * 256 >= vdim
template <typename T, int NR>
__global__ void __launch_bounds__(256) grouped_decode_kernel(const GroupedParams p) {
  extern __shared__ float gd_smem[];
  const int dp = p.dim + 1;
  float* qs = gd_smem;                 // [GD_HEADS][dim + 1]
  float* ks = qs + GD_HEADS * dp;      // [GD_KEYS][dim + 1]
  float* vs = ks + GD_KEYS * dp;       // [GD_KEYS][vdim]
  __shared__ float sc[GD_HEADS][GD_KEYS], resc[GD_HEADS], ms[GD_HEADS], ls[GD_HEADS];
  const int per = p.H / p.G, tiles = (per + GD_HEADS - 1) / GD_HEADS;
  const int b = blockIdx.z, g = blockIdx.y / tiles, sp = blockIdx.x, tid = threadIdx.x;
  const int h0 = g * per + (blockIdx.y % tiles) * GD_HEADS, nh = min(GD_HEADS, (g + 1) * per - h0);
  int len = p.lengths[b];
  if (len < 0 || len > p.Tmax) {       // a length that does not fit the cache: never read past it
    if (tid == 0) OSLO_REPORT_BOUNDS(p.err);
    len = len < 0 ? 0 : p.Tmax;
  }
  const int span = (len + p.splits - 1) / p.splits;
  const int t0 = sp * span, t1 = min(len, t0 + span);
  const T* q = static_cast<const T*>(p.q) + (static_cast<long long>(b) * p.H + h0) * p.dim;
  for (int e = tid; e < GD_HEADS * p.dim; e += 256) {
    const int a = e / p.dim, c = e - a * p.dim;
    qs[a * dp + c] = a < nh ? Num<T>::to(q[e]) * p.scale : 0.f;
  }
  if (tid < GD_HEADS) { ms[tid] = -CUDART_INF_F; ls[tid] = 0.f; }
  float acc[NR][GD_HEADS];
#pragma unroll
  for (int j = 0; j < NR; ++j)
#pragma unroll
    for (int a = 0; a < GD_HEADS; ++a) acc[j][a] = 0.f;
  const T* kb = static_cast<const T*>(p.kc) + (static_cast<long long>(b) * p.G + g) * p.Tmax * p.dim;
  const T* vb = static_cast<const T*>(p.vc) + (static_cast<long long>(b) * p.G + g) * p.Tmax * p.vdim;
  for (int k0 = t0; k0 < t1; k0 += GD_KEYS) {
    const int n = min(GD_KEYS, t1 - k0);
    __syncthreads();
    for (int e = tid; e < GD_KEYS * p.dim; e += 256) {
      const int t = e / p.dim, c = e - t * p.dim;
      ks[t * dp + c] = t < n ? Num<T>::to(kb[static_cast<long long>(k0) * p.dim + e]) : 0.f;
    }
    for (int e = tid; e < GD_KEYS * p.vdim; e += 256)
      vs[e] = e < n * p.vdim ? Num<T>::to(vb[static_cast<long long>(k0) * p.vdim + e]) : 0.f;
    __syncthreads();
    {
      const int a = tid >> 5, t = tid & 31;              // warp = head, lane = key
      float d = 0.f;
      for (int c = 0; c < p.dim; ++c) d = fmaf(qs[a * dp + c], ks[t * dp + c], d);
      if (p.softcap > 0.f) d = p.softcap * tanhf(d / p.softcap);
      const int pos = k0 + t;
      const bool vis = t < n && (p.keep == nullptr || pos >= p.n_keep || p.keep[b * p.ld_keep + pos]);
      d = vis ? d : -CUDART_INF_F;
      float mx = d;
#pragma unroll
      for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
      const float m_old = ms[a], m_new = fmaxf(m_old, mx);
      const float e = d == -CUDART_INF_F ? 0.f : expf(d - m_new);
      const float s = warp_sum(e);
      sc[a][t] = e;
      if (t == 0) {
        const float f = m_old == -CUDART_INF_F ? 0.f : expf(m_old - m_new);
        resc[a] = f;
        ls[a] = ls[a] * f + s;
      }
      __syncwarp();
      if (t == 0) ms[a] = m_new;
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < NR; ++j) {
      const int c = tid + j * 256;
      if (c < p.vdim) {
#pragma unroll
        for (int a = 0; a < GD_HEADS; ++a) acc[j][a] *= resc[a];
#pragma unroll 4
        for (int t = 0; t < GD_KEYS; ++t) {
          const float x = vs[t * p.vdim + c];
#pragma unroll
          for (int a = 0; a < GD_HEADS; ++a) acc[j][a] = fmaf(sc[a][t], x, acc[j][a]);
        }
      }
    }
  }
  __syncthreads();
  for (int a = 0; a < nh; ++a) {
    const long long at = (static_cast<long long>(b) * p.H + h0 + a) * p.splits + sp;
#pragma unroll
    for (int j = 0; j < NR; ++j) {
      const int c = tid + j * 256;
      if (c < p.vdim) {
        float v = 0.f;
#pragma unroll
        for (int u = 0; u < GD_HEADS; ++u) v = u == a ? acc[j][u] : v;
        p.ws[at * p.ldw + c] = v;
      }
    }
    if (tid == 0) { p.stat[at * 2] = ms[a]; p.stat[at * 2 + 1] = ls[a]; }
  }
}

// block = (head, row): merge the slices; exp(sink) joins the denominator
template <typename T>
__global__ void __launch_bounds__(128) grouped_finish_kernel(const float* __restrict__ ws, const float* __restrict__ stat,
                                                             const T* __restrict__ sink, T* __restrict__ out, int H, int vdim,
                                                             int ldw, int splits) {
  const int h = blockIdx.x, b = blockIdx.y;
  const long long at = (static_cast<long long>(b) * H + h) * splits;
  float m = Num<T>::to(sink[h]);
  for (int s = 0; s < splits; ++s) m = fmaxf(m, stat[(at + s) * 2]);
  float tot = expf(Num<T>::to(sink[h]) - m);
  for (int s = 0; s < splits; ++s) {
    const float ms = stat[(at + s) * 2];
    if (ms != -CUDART_INF_F) tot = fmaf(stat[(at + s) * 2 + 1], expf(ms - m), tot);
  }
  const float inv = 1.0f / tot;
  for (int c = threadIdx.x; c < vdim; c += blockDim.x) {
    float v = 0.f;
    for (int s = 0; s < splits; ++s) {
      const float ms = stat[(at + s) * 2];
      if (ms != -CUDART_INF_F) v = fmaf(ws[(at + s) * ldw + c], expf(ms - m), v);
    }
    out[(static_cast<long long>(b) * H + h) * vdim + c] = Num<T>::from(v * inv);
  }
}

}  // namespace oslo

extern "C" int oslo_qkv_prep(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv,
                             const void* wq, const void* wk, float eps, const long long* pos, long long pos_sb, long long pos_ss,
                             const float* freq, int n_freq, void* q_out, void* kc, void* vc, const int* lengths, int B, int S,
                             int H, int G, int dim, int vdim, int Tmax, int dtype, int* err_word, cudaStream_t stream) {
  using namespace oslo;
  if (B <= 0 || S <= 0) return 0;
  if (H <= 0 || G <= 0 || dim <= 0 || vdim <= 0 || 2 * n_freq > dim) return -1;
  PrepParams p{q, k, v, ldq, ldk, ldv, wq, wk, pos, pos_sb, pos_ss, freq, n_freq, q_out, kc, vc, lengths, S, H, G, dim, vdim,
               Tmax, static_cast<long long>(B) * S * (H + 2 * G), eps, err_word};
  const long long blocks = (p.slots + 7) / 8;
  if (blocks > 0x7fffffffll) return -1;
  OSLO_DISPATCH_T(dtype, { qkv_prep_kernel<T><<<static_cast<unsigned>(blocks), 256, 0, stream>>>(p); });
  return static_cast<int>(cudaGetLastError());
}

extern "C" int oslo_grouped_splits(int B, int H, int G, int T, int num_sms) {
  const int tiles = (H / G + oslo::GD_HEADS - 1) / oslo::GD_HEADS;
  const long long blocks = static_cast<long long>(B) * G * tiles;
  long long s = (3ll * num_sms + blocks - 1) / blocks;
  s = std::min<long long>(s, (T + 127) / 128);           // a slice keeps at least 128 positions of a full cache
  return static_cast<int>(std::max<long long>(1, std::min<long long>(s, 128)));
}

extern "C" int oslo_grouped_decode(const void* q, const void* kc, const void* vc, const int* lengths, const uint8_t* keep,
                                   long long ld_keep, int n_keep, const void* sink, float* ws, float* stat, void* out, int B,
                                   int H, int G, int dim, int vdim, int Tmax, int splits, float scale, float softcap, int dtype,
                                   int* err_word, cudaStream_t stream) {
  using namespace oslo;
  if (B <= 0 || H <= 0) return 0;
  if (G <= 0 || H % G || B > 65535 || splits < 1) return -1;
  GroupedParams p{q, kc, vc, lengths, keep, ld_keep, n_keep, ws, stat, H, G, dim, vdim, (vdim + 3) / 4 * 4, Tmax, splits,
                  scale, softcap, err_word};
  const int tiles = (H / G + GD_HEADS - 1) / GD_HEADS;
  const dim3 grid(splits, G * tiles, B);
  const size_t smem = (static_cast<size_t>(GD_HEADS + GD_KEYS) * (dim + 1) + static_cast<size_t>(GD_KEYS) * vdim) * sizeof(float);
  if (smem > 220 * 1024 || static_cast<long long>(G) * tiles > 65535) return -3;
#define GD_GO(NR)                                                                                                  \
  {                                                                                                                \
    if (smem > 40 * 1024) {                                                                                        \
      cudaError_t e = cudaFuncSetAttribute(grouped_decode_kernel<T, NR>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                           static_cast<int>(smem));                                                \
      if (e != cudaSuccess) return static_cast<int>(e);                                                            \
    }                                                                                                              \
    grouped_decode_kernel<T, NR><<<grid, 256, smem, stream>>>(p);                                                  \
  }
  OSLO_DISPATCH_T(dtype, {
    if (vdim <= 256) GD_GO(1)
    else if (vdim <= 512) GD_GO(2)
    else if (vdim <= 1024) GD_GO(4)
    else return -3;
    grouped_finish_kernel<T><<<dim3(H, B), 128, 0, stream>>>(ws, stat, static_cast<const T*>(sink), static_cast<T*>(out), H, vdim,
                                                             p.ldw, splits);
  });
#undef GD_GO
  return static_cast<int>(cudaGetLastError());
}
