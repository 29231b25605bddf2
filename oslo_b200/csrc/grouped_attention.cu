// Grouped-query attention with query / key norms, rotation, capped scores, a sink in the denominator, a window that
// keeps the first keys and an output gate per head or element:
// what comes before the scores (qkv_prep_kernel, head_prep_kernel) and decoding with one query per row (grouped_decode_kernel). Prompts
// run on the tcgen05 flash kernels (attention_sm100.cu) or, in 32-bit, on sink_attention_kernel (latent_attention.cu).
//
// Talking heads: scores mixed over the heads before the softmax, score_h <- sum_g talk[h, g] q_g . k_{group(g)}, are products of one
// wide key per token (all key heads in a row) with the query [sum_{g in group 0} talk[h, g] q_g | the same of group 1 | ...].
// head_prep_kernel writes these queries from normed and rotated heads in 32-bit, rounding once; from there on it is attention
// with one key head for all query heads and value heads per group (wide_decode_kernel; fa_wide_kernel for prompts).
//
// Decode: a block scans a slice of one key / value head's cache for the query heads that share it (up to 16 on tensor cores,
// 8 in the 32-bit version), so every cached byte is read once per block; grouped_finish_kernel merges the slices, adds the
// sink to the denominator and gates. With a window the slices run over the visible keys only (KeyRun).
#include <math_constants.h>

#include <algorithm>

#include "num.cuh"
#include "oslo_kernels.h"
#include "ptx.cuh"

namespace oslo {

// ------------------------------------------------------------------ norms, rotation, cache append
struct PrepParams {
  const void *q, *k, *v; long long ldq, ldk, ldv;     // row b * S + t
  const void *wq, *wk;                                // [dim], or nullptr: norms without a weight
  const long long* pos; long long pos_sb, pos_ss;
  const float* freq; int n_freq;
  void *q_out, *kc, *vc;                              // [B, S, H, dim], [B, G, Tmax, dim], [B, G, Tmax, vdim]
  const int* lengths;
  int S, H, G, dim, vdim, Tmax;
  long long slots;                                    // B * S * (H + 2 G)
  float eps;
  int* err;
};

// one warp per (token, head): H query heads, G key heads, G value heads; VEC 4: rows and head slices are aligned to four elements
template <typename T, int VEC>
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
      for (int c = lane * VEC; c < p.vdim; c += 32 * VEC)
        *reinterpret_cast<Pack<T, VEC>*>(dst + c) = *reinterpret_cast<const Pack<T, VEC>*>(src + c);
      return;
    }
    src = static_cast<const T*>(p.k) + row * p.ldk + static_cast<long long>(h) * p.dim;
    dst = static_cast<T*>(p.kc) + ((b * p.G + h) * p.Tmax + at) * p.dim;
  }
  const T* w = static_cast<const T*>(is_q ? p.wq : p.wk);
  const float at = static_cast<float>(p.pos[b * p.pos_sb + t * p.pos_ss]);
  if constexpr (VEC == 4) {
    if (p.dim <= 256) {                                // the head stays in registers: at most two groups of four per lane
      float x[2][4], ss = 0.f;
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int c = 4 * (lane + 32 * u);
        if (c < p.dim) {
          load_vec<T, 4>(src + c, x[u]);
#pragma unroll
          for (int i = 0; i < 4; ++i) ss = fmaf(x[u][i], x[u][i], ss);
        }
      }
      const float r = 1.0f / sqrtf(warp_sum(ss) / p.dim + p.eps);
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int c = 4 * (lane + 32 * u);
        if (c >= p.dim) break;
        float g[4] = {1.f, 1.f, 1.f, 1.f};
        if (w != nullptr) load_vec<T, 4>(w + c, g);
#pragma unroll
        for (int i = 0; i < 4; ++i) x[u][i] *= r * g[i];
#pragma unroll
        for (int i = 0; i < 4; i += 2) {
          if (((c + i) >> 1) >= p.n_freq) continue;
          float sn, cs;
          sincosf(at * p.freq[(c + i) >> 1], &sn, &cs);
          const float v = x[u][i] * cs - x[u][i + 1] * sn;
          x[u][i + 1] = x[u][i + 1] * cs + x[u][i] * sn;
          x[u][i] = v;
        }
        store_vec<T, 4>(dst + c, x[u]);
      }
      return;
    }
  }
  float ss = 0.f;
  for (int c = lane; c < p.dim; c += 32) {
    const float x = Num<T>::to(src[c]);
    ss = fmaf(x, x, ss);
  }
  const float r = 1.0f / sqrtf(warp_sum(ss) / p.dim + p.eps);
  for (int c = 2 * lane; c < p.dim; c += 64) {         // the pair (c, c + 1)
    const bool two = c + 1 < p.dim;
    float x = Num<T>::to(src[c]) * r * (w ? Num<T>::to(w[c]) : 1.f);
    float y = two ? Num<T>::to(src[c + 1]) * r * (w ? Num<T>::to(w[c + 1]) : 1.f) : 0.f;
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

// ------------------------------------------------------------------ rotation by halves, queries of talking heads
struct HeadPrepParams {
  const void *q, *k, *v; long long ldq, ldk, ldv;     // row b * S + t
  const void *wq, *wk;                                // [dim], or nullptr
  const long long* pos; long long pos_sb, pos_ss;
  const float* freq; int n_freq, halves;
  float amplitude;                                    // of sines and cosines
  const void* talk;                                   // [H, H], or nullptr: the heads as they are
  void* q_out;                                        // [B, S, H, talk ? G * dim : dim]
  void *kc, *vc;                                      // heads g, position t at b * sb + g * sg + t * st
  long long k_sb, k_sg, k_st, v_sb, v_sg, v_st;
  const int* lengths;
  int S, H, G, dim, vdim, Tmax;
  float eps;
  int* err;
};

constexpr int HP_WARPS = 8;

// what heads h0..h1 of a token ask of the keys of all key heads: sums of the heads `qs` [H][dim] weighted by `ts` [h1 - h0][H]. PER: query
// heads per key head, 0: any number
template <typename T, int VEC, int PER>
__device__ __forceinline__ void head_mix(const HeadPrepParams& p, const float* qs, const float* ts, long long row, int h0, int h1) {
  const int H = p.H, dim = p.dim, per = PER > 0 ? PER : H / p.G, cols = p.G * dim, groups = cols / VEC;
  const int threads = static_cast<int>(blockDim.x), tid = threadIdx.x;
  T* out = static_cast<T*>(p.q_out) + (row * H + h0) * cols;
  // a thread owns VEC columns; with fewer columns than threads several threads share them, each with heads of its own
  const int lanes = groups < threads ? threads / groups : 1, step = groups < threads ? groups : threads;
  const int first = groups < threads ? tid / groups : 0;
  if (first >= lanes) return;
  for (int u = groups < threads ? tid - first * groups : tid; u < groups; u += step) {
    const int c = u * VEC, g = c / dim;
    const float* src = qs + g * per * dim + (c - g * dim);
    float x[PER > 0 ? PER : 1][VEC];
    if constexpr (PER > 0) {
#pragma unroll
      for (int r = 0; r < PER; ++r) load_vec<float, VEC>(src + r * dim, x[r]);
    }
    const float* tw = ts + first * H + g * per;
    T* dst = out + static_cast<long long>(first) * cols + c;
#pragma unroll 2
    for (int h = first; h < h1 - h0; h += lanes, tw += lanes * H, dst += static_cast<long long>(lanes) * cols) {
      float o[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) o[i] = 0.f;
      if constexpr (PER > 0) {
        constexpr int W = PER % 4 == 0 ? 4 : 1;        // weights read at a time; H is a multiple of PER
#pragma unroll
        for (int r = 0; r < PER; r += W) {
          float m[W];
          load_vec<float, W>(tw + r, m);
#pragma unroll
          for (int k = 0; k < W; ++k)
#pragma unroll
            for (int i = 0; i < VEC; ++i) o[i] = fmaf(m[k], x[r + k][i], o[i]);
        }
      } else {
        for (int r = 0; r < per; ++r) {
          float y[VEC];
          load_vec<float, VEC>(src + r * dim, y);
#pragma unroll
          for (int i = 0; i < VEC; ++i) o[i] = fmaf(tw[r], y[i], o[i]);
        }
      }
      store_vec<T, VEC>(dst, o);
    }
  }
}

// block = (token, share of the query heads that are written); the first share also does keys and values. Angles are
// computed once per token. VEC 4: everything is aligned to four elements
template <typename T, int VEC>
__global__ void __launch_bounds__(32 * HP_WARPS) head_prep_kernel(const HeadPrepParams p) {
  extern __shared__ float hp_smem[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, H = p.H, dim = p.dim;
  float* cs = hp_smem;                                 // [n_freq]
  float* sn = cs + p.n_freq;                           // [n_freq]
  float* qs = sn + p.n_freq + (2 * p.n_freq % 4 ? 4 - 2 * p.n_freq % 4 : 0);   // [talk ? H : HP_WARPS][dim], 16-byte aligned
  float* kb = qs + (p.talk ? H : HP_WARPS) * dim;      // [HP_WARPS][dim]
  float* ts = kb + HP_WARPS * dim;                     // [share][H]
  const long long row = blockIdx.x;
  const long long b = row / p.S, t = row - b * p.S;
  const int share = (H + gridDim.y - 1) / gridDim.y, h0 = blockIdx.y * share, h1 = min(H, h0 + share);
  const float at = static_cast<float>(p.pos[b * p.pos_sb + t * p.pos_ss]);
  for (int i = tid; i < p.n_freq; i += blockDim.x) {
    float s, c;
    sincosf(at * p.freq[i], &s, &c);
    cs[i] = c * p.amplitude;
    sn[i] = s * p.amplitude;
  }
  if (p.talk != nullptr)
    for (int e = tid; e < (h1 - h0) * H; e += blockDim.x) ts[e] = Num<T>::to(static_cast<const T*>(p.talk)[static_cast<long long>(h0) * H + e]);
  __syncthreads();
  // one head, normed and rotated, in `buf`
  auto head = [&](const T* src, const T* w, float* buf) {
    float ss = 0.f;
    for (int c = lane * VEC; c < dim; c += 32 * VEC) {
      float x[VEC];
      load_vec<T, VEC>(src + c, x);
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss = fmaf(x[i], x[i], ss);
      store_vec<float, VEC>(buf + c, x);
    }
    const float r = 1.0f / sqrtf(warp_sum(ss) / dim + p.eps);
    __syncwarp();
    const int n = p.n_freq;
#pragma unroll 2
    for (int i = lane; i < n; i += 32) {               // pairs
      const int a = p.halves ? i : 2 * i, c = p.halves ? i + n : 2 * i + 1;
      const float x = buf[a] * r * (w ? Num<T>::to(w[a]) : 1.f), y = buf[c] * r * (w ? Num<T>::to(w[c]) : 1.f);
      buf[a] = x * cs[i] - y * sn[i];
      buf[c] = y * cs[i] + x * sn[i];
    }
    for (int c = 2 * n + lane; c < dim; c += 32) buf[c] *= r * (w ? Num<T>::to(w[c]) : 1.f);
    __syncwarp();
  };
  auto put = [&](T* dst, const float* buf) {
    for (int c = lane * VEC; c < dim; c += 32 * VEC) {
      float x[VEC];
      load_vec<float, VEC>(buf + c, x);
      store_vec<T, VEC>(dst + c, x);
    }
  };
  const T* q = static_cast<const T*>(p.q) + row * p.ldq;
  const int q0 = p.talk ? 0 : h0, q1 = p.talk ? H : h1;
  for (int h = q0 + warp; h < q1; h += HP_WARPS) {
    float* buf = qs + (p.talk ? h : warp) * dim;
    head(q + static_cast<long long>(h) * dim, static_cast<const T*>(p.wq), buf);
    if (p.talk == nullptr) {
      put(static_cast<T*>(p.q_out) + (row * H + h) * dim, buf);
      __syncwarp();
    }
  }
  if (blockIdx.y == 0) {
    const long long to = p.lengths[b] + t;
    if (to < 0 || to >= p.Tmax) {                      // never write outside the cache
      if (tid == 0) OSLO_REPORT_BOUNDS(p.err);
    } else {
      for (int g = warp; g < 2 * p.G; g += HP_WARPS) {
        if (g < p.G) {
          float* buf = kb + warp * dim;
          head(static_cast<const T*>(p.k) + row * p.ldk + static_cast<long long>(g) * dim, static_cast<const T*>(p.wk), buf);
          put(static_cast<T*>(p.kc) + b * p.k_sb + g * p.k_sg + to * p.k_st, buf);
          __syncwarp();
        } else {
          const T* src = static_cast<const T*>(p.v) + row * p.ldv + static_cast<long long>(g - p.G) * p.vdim;
          T* dst = static_cast<T*>(p.vc) + b * p.v_sb + (g - p.G) * p.v_sg + to * p.v_st;
          for (int c = lane * VEC; c < p.vdim; c += 32 * VEC)
            *reinterpret_cast<Pack<T, VEC>*>(dst + c) = *reinterpret_cast<const Pack<T, VEC>*>(src + c);
        }
      }
    }
  }
  if (p.talk == nullptr) return;
  __syncthreads();
  const int per = H / p.G;
  if (per == 4 && VEC == 4) head_mix<T, VEC, 4>(p, qs, ts, row, h0, h1);
  else if (per == 8 && VEC == 4) head_mix<T, VEC, 8>(p, qs, ts, row, h0, h1);
  else if (per == 2) head_mix<T, VEC, 2>(p, qs, ts, row, h0, h1);
  else if (per == 1) head_mix<T, VEC, 1>(p, qs, ts, row, h0, h1);
  else head_mix<T, VEC, 0>(p, qs, ts, row, h0, h1);
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
  int VG;                              // value heads in a cached value row (wide keys: G = 1, all value heads in a row); else 1
  float scale, softcap;
  int window, keep_first;              // window > 0: the last `window` positions, and the first keep_first after lead[b]
  const int* lead;                     // [B] padding ahead of the sequence, or nullptr
  int* err;
};

// the positions a query reads, as one run of `n` indices: `head` of them from `first`, the others up to the sequence's end
struct KeyRun {
  int first, head, jump, n;
  __device__ __forceinline__ KeyRun(const GroupedParams& p, int b, int len) {
    if (p.window <= 0 || p.window >= len) {
      first = 0; head = n = len; jump = 0;
      return;
    }
    const int tail = len - p.window;
    first = p.lead ? max(0, min(p.lead[b], tail)) : 0;
    head = min(p.keep_first, tail - first);
    jump = tail - (first + head);
    n = head + p.window;
  }
  __device__ __forceinline__ int at(int i) const { return first + i + (i >= head ? jump : 0); }
};

constexpr int GD_HEADS = 8, GD_KEYS = 32, GD_MAX_SPLITS = 128;

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
  const KeyRun run(p, b, len);
  const int span = (run.n + p.splits - 1) / p.splits;
  const int t0 = sp * span, t1 = min(run.n, t0 + span);
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
      ks[t * dp + c] = t < n ? Num<T>::to(kb[static_cast<long long>(run.at(k0 + t)) * p.dim + c]) : 0.f;
    }
    for (int e = tid; e < GD_KEYS * p.vdim; e += 256) {
      const int t = e / p.vdim, c = e - t * p.vdim;
      vs[e] = t < n ? Num<T>::to(vb[static_cast<long long>(run.at(k0 + t)) * p.vdim + c]) : 0.f;
    }
    __syncthreads();
    {
      const int a = tid >> 5, t = tid & 31;              // warp = head, lane = key
      float d = 0.f;
      for (int c = 0; c < p.dim; ++c) d = fmaf(qs[a * dp + c], ks[t * dp + c], d);
      if (p.softcap > 0.f) d = p.softcap * tanhf(d / p.softcap);
      const int pos = run.at(k0 + t);
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
  const int vd = p.vdim / p.VG;
  for (int a = 0; a < nh; ++a) {
    const long long at = (static_cast<long long>(b) * p.H + h0 + a) * p.splits + sp;
    const int own = p.VG > 1 ? (h0 + a) / (p.H / p.VG) * vd : 0;          // the head's own columns
#pragma unroll
    for (int j = 0; j < NR; ++j) {
      const int c = tid + j * 256 - own;
      if (c >= 0 && c < vd) {
        float v = 0.f;
#pragma unroll
        for (int u = 0; u < GD_HEADS; ++u) v = u == a ? acc[j][u] : v;
        p.ws[at * p.ldw + c] = v;
      }
    }
    if (tid == 0) { p.stat[at * 2] = ms[a]; p.stat[at * 2 + 1] = ls[a]; }
  }
}

// ------------------------------------------------------------------ decode, 16-bit heads on tensor cores
__device__ __forceinline__ void gd_ldsm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void gd_ldsm4_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
template <typename T> struct GdMma;
template <> struct GdMma<__nv_bfloat16> {
  static __device__ __forceinline__ void run(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
  }
  static __device__ __forceinline__ uint32_t pack(float x, float y) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    return *reinterpret_cast<const uint32_t*>(&h);
  }
};
template <> struct GdMma<__half> {
  static __device__ __forceinline__ void run(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
  }
  static __device__ __forceinline__ uint32_t pack(float x, float y) {
    const __half2 h = __floats2half2_rn(x, y);
    return *reinterpret_cast<const uint32_t*>(&h);
  }
};

constexpr float GD_LOG2E = 1.4426950408889634f, GD_LN2 = 0.6931471805599453f;
__device__ __forceinline__ float gd_exp2(float x) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}

constexpr int GM_HEADS = 16, GM_KEYS = 64;   // rows of a product; keys per stage, 16 of them per warp

template <int D> constexpr size_t gd_mma_smem() { return static_cast<size_t>(GM_HEADS + 4 * GM_KEYS) * (D + 8) * 2; }

// head sizes (multiples of 8) up to D; every warp keeps a softmax of its own over its keys, merged at the end
template <typename T, int D>
__global__ void __launch_bounds__(128) grouped_decode_mma_kernel(const GroupedParams p) {
  constexpr int PITCH = D + 8;
  extern __shared__ uint4 gm_smem[];
  T* qs = reinterpret_cast<T*>(gm_smem);     // [GM_HEADS][PITCH]
  T* ks = qs + GM_HEADS * PITCH;             // [2][GM_KEYS][PITCH]
  T* vs = ks + 2 * GM_KEYS * PITCH;          // [2][GM_KEYS][PITCH]
  __shared__ float ms[4][GM_HEADS], ls[4][GM_HEADS];
  const int per = p.H / p.G, tiles = (per + GM_HEADS - 1) / GM_HEADS;
  const int b = blockIdx.z, g = blockIdx.y / tiles, sp = blockIdx.x, tid = threadIdx.x, w = tid >> 5, l = tid & 31;
  const int h0 = g * per + (blockIdx.y % tiles) * GM_HEADS, nh = min(GM_HEADS, (g + 1) * per - h0);
  int len = p.lengths[b];
  if (len < 0 || len > p.Tmax) {             // a length that does not fit the cache: never read past it
    if (tid == 0) OSLO_REPORT_BOUNDS(p.err);
    len = len < 0 ? 0 : p.Tmax;
  }
  const KeyRun run(p, b, len);
  const int span = (run.n + p.splits - 1) / p.splits;
  const int t0 = sp * span, t1 = min(run.n, t0 + span);
  const T* kb = static_cast<const T*>(p.kc) + (static_cast<long long>(b) * p.G + g) * p.Tmax * p.dim;
  const T* vb = static_cast<const T*>(p.vc) + (static_cast<long long>(b) * p.G + g) * p.Tmax * p.vdim;
  // columns past the head sizes are zero for good: the copies below never write them
  for (int e = tid; e < (GM_HEADS + 4 * GM_KEYS) * PITCH / 8; e += 128) gm_smem[e] = make_uint4(0, 0, 0, 0);
  __syncthreads();
  const T* q = static_cast<const T*>(p.q) + (static_cast<long long>(b) * p.H + h0) * p.dim;
  for (int e = tid; e < nh * (p.dim / 8); e += 128) {
    const int a = e / (p.dim / 8), c = e % (p.dim / 8) * 8;
    *reinterpret_cast<uint4*>(qs + a * PITCH + c) = *reinterpret_cast<const uint4*>(q + a * p.dim + c);
  }
  // a thread copies the same 16-byte column of every `rows`-th key
  auto copy = [&](T* dst, const T* src, int width, int rows, int t_first, int c, int k0) {
    if (t_first >= rows) return;
#pragma unroll 4
    for (int t = t_first; t < GM_KEYS; t += rows) {
      const bool ok = k0 + t < t1;
      const uint32_t d32 = smem_u32(dst + t * PITCH + c);
      const int bytes = ok ? 16 : 0;         // 0: the 16 bytes are filled with zeros
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d32), "l"(src + static_cast<long long>(run.at(ok ? k0 + t : t0)) * width + c), "r"(bytes) : "memory");
    }
  };
  const int k_rows = 128 / (p.dim / 8), k_first = tid / (p.dim / 8), k_col = tid % (p.dim / 8) * 8;
  const int v_rows = 128 / (p.vdim / 8), v_first = tid / (p.vdim / 8), v_col = tid % (p.vdim / 8) * 8;
  auto fetch = [&](int k0, int buf) {
    copy(ks + buf * GM_KEYS * PITCH, kb, p.dim, k_rows, k_first, k_col, k0);
    copy(vs + buf * GM_KEYS * PITCH, vb, p.vdim, v_rows, v_first, v_col, k0);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  float o[D / 8][4];
#pragma unroll
  for (int i = 0; i < D / 8; ++i) { o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f; }
  float m[2] = {-CUDART_INF_F, -CUDART_INF_F}, s[2] = {0.f, 0.f};     // rows l / 4 and l / 4 + 8; scores in log2 units
  const float cap = p.softcap * GD_LOG2E, scale = p.softcap > 0.f ? 2.f * p.scale / p.softcap * GD_LOG2E : p.scale * GD_LOG2E;
  if (t0 < t1) fetch(t0, 0);
  for (int k0 = t0, it = 0; k0 < t1; k0 += GM_KEYS, ++it) {
    const int buf = it & 1;
    if (k0 + GM_KEYS < t1) {
      fetch(k0 + GM_KEYS, buf ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const T* kw = ks + (buf * GM_KEYS + w * 16) * PITCH;
    const T* vw = vs + (buf * GM_KEYS + w * 16) * PITCH;
    float c[2][4] = {};
#pragma unroll
    for (int kk = 0; kk < D / 16; ++kk) {
      uint32_t a[4], bb[4];
      gd_ldsm4(a, smem_u32(qs + ((l & 7) + ((l >> 3) & 1) * 8) * PITCH + kk * 16 + (l >> 4) * 8));
      gd_ldsm4(bb, smem_u32(kw + ((l & 7) + (l >> 4) * 8) * PITCH + kk * 16 + ((l >> 3) & 1) * 8));
      GdMma<T>::run(c[0], a, bb[0], bb[1]);
      GdMma<T>::run(c[1], a, bb[2], bb[3]);
    }
    float mx[2] = {m[0], m[1]};
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = k0 + w * 16 + nt * 8 + (l & 3) * 2 + (e & 1), pos = run.at(i);
        const bool vis = i < t1 && (p.keep == nullptr || pos >= p.n_keep || p.keep[b * p.ld_keep + pos]);
        float d = c[nt][e] * scale;                    // capped: twice the score over the cap, in log2 units
        if (p.softcap > 0.f) d = cap - __fdividef(2.f * cap, gd_exp2(d) + 1.f);   // cap * tanh(score / cap)
        c[nt][e] = vis ? d : -CUDART_INF_F;
        mx[e >> 1] = fmaxf(mx[e >> 1], c[nt][e]);
      }
    }
    float alpha[2], ref[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
      mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
      ref[i] = mx[i] == -CUDART_INF_F ? 0.f : mx[i];
      alpha[i] = gd_exp2(m[i] - ref[i]);               // 2^-inf = 0
      m[i] = mx[i];
      s[i] *= alpha[i];
    }
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        c[nt][e] = gd_exp2(c[nt][e] - ref[e >> 1]);
        s[e >> 1] += c[nt][e];
      }
    }
    if (__any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f)) {
#pragma unroll
      for (int i = 0; i < D / 8; ++i) { o[i][0] *= alpha[0]; o[i][1] *= alpha[0]; o[i][2] *= alpha[1]; o[i][3] *= alpha[1]; }
    }
    const uint32_t pf[4] = {GdMma<T>::pack(c[0][0], c[0][1]), GdMma<T>::pack(c[0][2], c[0][3]), GdMma<T>::pack(c[1][0], c[1][1]),
                            GdMma<T>::pack(c[1][2], c[1][3])};
#pragma unroll
    for (int dt = 0; dt < D / 8; dt += 2) {
      uint32_t bb[4];
      gd_ldsm4_t(bb, smem_u32(vw + ((l & 7) + ((l >> 3) & 1) * 8) * PITCH + dt * 8 + (l >> 4) * 8));
      GdMma<T>::run(o[dt], pf, bb[0], bb[1]);
      GdMma<T>::run(o[dt + 1], pf, bb[2], bb[3]);
    }
    __syncthreads();                                   // the stage may be fetched over
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    s[i] += __shfl_xor_sync(0xffffffffu, s[i], 1);
    s[i] += __shfl_xor_sync(0xffffffffu, s[i], 2);
    if ((l & 3) == 0) { ms[w][(l >> 2) + 8 * i] = m[i]; ls[w][(l >> 2) + 8 * i] = s[i]; }
  }
  __syncthreads();                                     // no copies are in flight: the stages become [4][GM_HEADS][D] floats
  float* red = reinterpret_cast<float*>(ks);
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int row = (l >> 2) + 8 * i;
    const float top = fmaxf(fmaxf(ms[0][row], ms[1][row]), fmaxf(ms[2][row], ms[3][row]));
    const float f = m[i] == -CUDART_INF_F ? 0.f : gd_exp2(m[i] - top);
#pragma unroll
    for (int dt = 0; dt < D / 8; ++dt)
      *reinterpret_cast<float2*>(red + (w * GM_HEADS + row) * D + dt * 8 + (l & 3) * 2) = make_float2(o[dt][2 * i] * f, o[dt][2 * i + 1] * f);
  }
  __syncthreads();
  for (int e = tid; e < nh * p.vdim; e += 128) {
    const int a = e / p.vdim, c = e - a * p.vdim;
    const long long at = (static_cast<long long>(b) * p.H + h0 + a) * p.splits + sp;
    p.ws[at * p.ldw + c] = red[a * D + c] + red[(GM_HEADS + a) * D + c] + red[(2 * GM_HEADS + a) * D + c] + red[(3 * GM_HEADS + a) * D + c];
  }
  if (tid < nh) {
    const float top = fmaxf(fmaxf(ms[0][tid], ms[1][tid]), fmaxf(ms[2][tid], ms[3][tid]));
    float tot = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) tot += ms[i][tid] == -CUDART_INF_F ? 0.f : ls[i][tid] * gd_exp2(ms[i][tid] - top);
    const long long at = (static_cast<long long>(b) * p.H + h0 + tid) * p.splits + sp;
    p.stat[at * 2] = top * GD_LN2;
    p.stat[at * 2 + 1] = tot;
  }
}

// ------------------------------------------------------------------ decode, wide keys on tensor cores
// One cached key row (dim columns) for all query heads, value heads side by side in a cached value row: block = (slice, up to 16 MT
// query heads, row). A stage of KEYS keys and values is on its way while the one before is used: (1) scores of 16 heads x 16 keys per
// warp (over a share of the columns when there are fewer tiles than warps), (2) softmax, head rows dealt out to the warps, (3) 16 heads x
// 32 value columns per item, only the columns of these heads' groups.
constexpr int WD_WARPS = 16, WD_COLS = 32;

struct WideLayout {
  int kp, vp;                          // row pitches of the key and value stages
  size_t q, k, v, s, p, total;         // byte offsets
};
template <int MT, int KEYS, int NBUF>
__host__ __device__ inline WideLayout wide_layout(int dim, int vdim) {
  WideLayout l;
  l.kp = (dim + 15) / 16 * 16 + 8;     // 16-byte rows whose starts fall on different banks
  l.vp = (vdim + 15) / 16 * 16 + 8;
  constexpr int TILES = MT * KEYS / 16, KSPLIT = WD_WARPS / TILES;
  l.q = 0;
  l.k = l.q + static_cast<size_t>(MT) * 16 * l.kp * 2;
  l.v = l.k + static_cast<size_t>(NBUF) * KEYS * l.kp * 2;
  l.s = l.v + static_cast<size_t>(NBUF) * KEYS * l.vp * 2;
  l.p = l.s + static_cast<size_t>(KSPLIT) * MT * 16 * (KEYS + 1) * 4;
  l.p = (l.p + 15) / 16 * 16;
  l.total = l.p + static_cast<size_t>(MT) * 16 * (KEYS + 8) * 2;
  return l;
}

template <typename T, int MT, int KEYS, int NBUF, int ITEMS>
__global__ void __launch_bounds__(32 * WD_WARPS) wide_decode_kernel(const GroupedParams p) {
  constexpr int ROWS = MT * 16, TILES = MT * KEYS / 16, KSPLIT = WD_WARPS / TILES;
  constexpr int RW = ROWS / WD_WARPS;                  // head rows of a warp in step 2
  static_assert(TILES * KSPLIT == WD_WARPS && RW * WD_WARPS == ROWS && KEYS <= 32, "a warp has one share of a tile of scores, a lane one key");
  extern __shared__ uint4 gm_smem[];
  const WideLayout lay = wide_layout<MT, KEYS, NBUF>(p.dim, p.vdim);
  uint8_t* base = reinterpret_cast<uint8_t*>(gm_smem);
  T* qs = reinterpret_cast<T*>(base + lay.q);          // [ROWS][kp]
  T* ks = reinterpret_cast<T*>(base + lay.k);          // [NBUF][KEYS][kp]
  T* vs = reinterpret_cast<T*>(base + lay.v);          // [NBUF][KEYS][vp]
  float* sc = reinterpret_cast<float*>(base + lay.s);  // [KSPLIT][ROWS][KEYS + 1]
  T* ps = reinterpret_cast<T*>(base + lay.p);          // [ROWS][KEYS + 8]
  __shared__ float alpha_s[ROWS];
  const int b = blockIdx.z, sp = blockIdx.x, tid = threadIdx.x, w = tid >> 5, l = tid & 31;
  const int h0 = blockIdx.y * ROWS, nh = min(ROWS, p.H - h0);
  const int vd = p.vdim / p.VG, per = p.H / p.VG;      // columns of a value head, query heads that read it
  int len = p.lengths[b];
  if (len < 0 || len > p.Tmax) {             // a length that does not fit the cache: never read past it
    if (tid == 0) OSLO_REPORT_BOUNDS(p.err);
    len = len < 0 ? 0 : p.Tmax;
  }
  const KeyRun run(p, b, len);
  const int span = (run.n + p.splits - 1) / p.splits;
  const int t0 = sp * span, t1 = min(run.n, t0 + span);
  const T* kb = static_cast<const T*>(p.kc) + static_cast<long long>(b) * p.Tmax * p.dim;
  const T* vb = static_cast<const T*>(p.vc) + static_cast<long long>(b) * p.Tmax * p.vdim;
  const T* q = static_cast<const T*>(p.q) + (static_cast<long long>(b) * p.H + h0) * p.dim;
  const int kc8 = p.dim / 8, vc8 = p.vdim / 8;
  // columns past the rows' ends and rows past the heads are zero for good: the copies below never write them
  for (int e = tid; e < ROWS * (lay.kp / 8); e += blockDim.x) {
    const int a = e / (lay.kp / 8), c = e % (lay.kp / 8);
    uint4 v = make_uint4(0, 0, 0, 0);
    if (a < nh && c < kc8) v = *reinterpret_cast<const uint4*>(q + static_cast<long long>(a) * p.dim + c * 8);
    *reinterpret_cast<uint4*>(qs + a * lay.kp + c * 8) = v;
  }
  for (int t = tid; t < NBUF * KEYS; t += blockDim.x) {
    for (int c = kc8; c < lay.kp / 8; ++c) *reinterpret_cast<uint4*>(ks + t * lay.kp + c * 8) = make_uint4(0, 0, 0, 0);
    for (int c = vc8; c < lay.vp / 8; ++c) *reinterpret_cast<uint4*>(vs + t * lay.vp + c * 8) = make_uint4(0, 0, 0, 0);
  }
  // a warp copies whole rows
  auto fetch = [&](int k0, int buf) {
    for (int t = w; t < KEYS; t += WD_WARPS) {
      const bool ok = k0 + t < t1;
      const long long pos = run.at(ok ? k0 + t : t0);
      const int bytes = ok ? 16 : 0;                   // 0: the 16 bytes are filled with zeros
      T* kd = ks + (buf * KEYS + t) * lay.kp;
      T* vdst = vs + (buf * KEYS + t) * lay.vp;
#pragma unroll 4
      for (int c = l; c < kc8; c += 32)
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(kd + c * 8)), "l"(kb + pos * p.dim + c * 8), "r"(bytes) : "memory");
#pragma unroll 4
      for (int c = l; c < vc8; c += 32)
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(vdst + c * 8)), "l"(vb + pos * p.vdim + c * 8), "r"(bytes) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // step 1: tile of this warp and its share of the columns
  const int tile = w % TILES, mt = tile % MT, kt = tile / MT, part = w / TILES;
  const int steps = (p.dim + 15) / 16, step0 = steps * part / KSPLIT, step1 = steps * (part + 1) / KSPLIT;
  // step 3: items (16 heads, WD_COLS of the columns of their groups), dealt out to the warps
  int item_mt[ITEMS], item_c0[ITEMS], item_c1[ITEMS];
#pragma unroll
  for (int i = 0; i < ITEMS; ++i) { item_mt[i] = -1; item_c0[i] = item_c1[i] = 0; }
  {
    int n = 0;
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      if (m * 16 >= nh) break;
      const int lo = (h0 + m * 16) / per * vd, hi = ((h0 + min(nh, m * 16 + 16) - 1) / per + 1) * vd;
      for (int c = lo; c < hi; c += WD_COLS, ++n)
        if (n % WD_WARPS == w) {
#pragma unroll
          for (int i = 0; i < ITEMS; ++i)
            if (i == n / WD_WARPS) { item_mt[i] = m; item_c0[i] = c; item_c1[i] = min(hi, c + WD_COLS); }
        }
    }
  }
  float o[ITEMS][WD_COLS / 8][4];
#pragma unroll
  for (int i = 0; i < ITEMS; ++i)
#pragma unroll
    for (int j = 0; j < WD_COLS / 8; ++j) o[i][j][0] = o[i][j][1] = o[i][j][2] = o[i][j][3] = 0.f;
  float m_row[RW], l_row[RW];                          // of the warp's head rows, the same in every lane; scores in log2 units
#pragma unroll
  for (int r = 0; r < RW; ++r) { m_row[r] = -CUDART_INF_F; l_row[r] = 0.f; }
  const float scale = p.scale * GD_LOG2E;
  const uint32_t qa = smem_u32(qs + mt * 16 * lay.kp + ((l & 7) + ((l >> 3) & 1) * 8) * lay.kp + (l >> 4) * 8);
  const uint32_t ka = smem_u32(ks + kt * 16 * lay.kp + ((l & 7) + (l >> 4) * 8) * lay.kp + ((l >> 3) & 1) * 8);
  const uint32_t k_stage = KEYS * lay.kp * 2;
  if (t0 < t1) fetch(t0, 0);
  for (int k0 = t0, it = 0; k0 < t1; k0 += KEYS, ++it) {
    const int buf = NBUF > 1 ? it & 1 : 0;
    if (NBUF > 1 && k0 + KEYS < t1) {
      fetch(k0 + KEYS, buf ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    {
      float c[2][4] = {};
      const uint32_t kaddr = ka + buf * k_stage;
#pragma unroll 4
      for (int kk = step0; kk < step1; ++kk) {
        uint32_t a[4], bb[4];
        gd_ldsm4(a, qa + kk * 32);
        gd_ldsm4(bb, kaddr + kk * 32);
        GdMma<T>::run(c[0], a, bb[0], bb[1]);
        GdMma<T>::run(c[1], a, bb[2], bb[3]);
      }
      float* dst = sc + (part * ROWS + mt * 16 + (l >> 2)) * (KEYS + 1) + kt * 16 + (l & 3) * 2;
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) dst[(e >> 1) * 8 * (KEYS + 1) + nt * 8 + (e & 1)] = c[nt][e];
    }
    __syncthreads();
    {
      const int pos = run.at(k0 + l);
      const bool vis = l < KEYS && k0 + l < t1 && (p.keep == nullptr || pos >= p.n_keep || p.keep[b * p.ld_keep + pos]);
#pragma unroll
      for (int r = 0; r < RW; ++r) {
        const int row = w * RW + r;
        float x = 0.f;
        if (l < KEYS) {
#pragma unroll
          for (int s = 0; s < KSPLIT; ++s) x += sc[(s * ROWS + row) * (KEYS + 1) + l];
        }
        const float d = vis ? x * scale : -CUDART_INF_F;
        float mx = d;
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
        mx = fmaxf(mx, m_row[r]);
        const float ref = mx == -CUDART_INF_F ? 0.f : mx, al = gd_exp2(m_row[r] - ref);     // 2^-inf = 0
        const float e = gd_exp2(d - ref);
        if (l < KEYS) ps[row * (KEYS + 8) + l] = Num<T>::from(e);
        if (l == 0) alpha_s[row] = al;
        l_row[r] = l_row[r] * al + warp_sum(e);
        m_row[r] = mx;
      }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      if (item_mt[i] < 0) continue;                    // uniform over the warp
      const float a0 = alpha_s[item_mt[i] * 16 + (l >> 2)], a1 = alpha_s[item_mt[i] * 16 + (l >> 2) + 8];
      if (__any_sync(0xffffffffu, a0 != 1.f || a1 != 1.f)) {
#pragma unroll
        for (int j = 0; j < WD_COLS / 8; ++j) { o[i][j][0] *= a0; o[i][j][1] *= a0; o[i][j][2] *= a1; o[i][j][3] *= a1; }
      }
      const T* pw = ps + item_mt[i] * 16 * (KEYS + 8);
#pragma unroll
      for (int kk = 0; kk < KEYS / 16; ++kk) {
        uint32_t a[4];
        gd_ldsm4(a, smem_u32(pw + ((l & 7) + ((l >> 3) & 1) * 8) * (KEYS + 8) + kk * 16 + (l >> 4) * 8));
        const T* vw = vs + (buf * KEYS + kk * 16 + (l & 7) + ((l >> 3) & 1) * 8) * lay.vp + item_c0[i] + (l >> 4) * 8;
#pragma unroll
        for (int j = 0; j < WD_COLS / 16; ++j) {
          if (item_c0[i] + j * 16 >= item_c1[i]) break;
          uint32_t bb[4];
          gd_ldsm4_t(bb, smem_u32(vw + j * 16));
          GdMma<T>::run(o[i][2 * j], a, bb[0], bb[1]);
          GdMma<T>::run(o[i][2 * j + 1], a, bb[2], bb[3]);
        }
      }
    }
    __syncthreads();                                   // the stage may be fetched over
    if (NBUF == 1 && k0 + KEYS < t1) fetch(k0 + KEYS, 0);
  }
#pragma unroll
  for (int i = 0; i < ITEMS; ++i) {
    if (item_mt[i] < 0) continue;
#pragma unroll
    for (int j = 0; j < WD_COLS / 8; ++j) {
      const int c = item_c0[i] + j * 8 + (l & 3) * 2;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int a = item_mt[i] * 16 + (l >> 2) + (e >> 1) * 8, col = c + (e & 1);
        if (a >= nh || col >= item_c1[i] || col / vd != (h0 + a) / per) continue;
        p.ws[((static_cast<long long>(b) * p.H + h0 + a) * p.splits + sp) * p.ldw + col % vd] = o[i][j][e];
      }
    }
  }
  if (l == 0) {
#pragma unroll
    for (int r = 0; r < RW; ++r) {
      const int a = w * RW + r;
      if (a >= nh) continue;
      const long long at = (static_cast<long long>(b) * p.H + h0 + a) * p.splits + sp;
      p.stat[at * 2] = m_row[r] * GD_LN2;
      p.stat[at * 2 + 1] = l_row[r];
    }
  }
}

constexpr size_t WD_SMEM = 220 * 1024;
// how the wide kernel runs these sizes: MT, KEYS, NBUF and ITEMS; keys 0: not at all
struct WidePlan { int mt, keys, nbuf, items; size_t smem; };
static WidePlan wide_plan(int H, int VG, int dim, int vdim, int dtype) {
  WidePlan w{0, 0, 0, 0, 0};
  if (dtype == OSLO_DT_FP32 || dim % 8 || vdim % VG || (vdim / VG) % 8) return w;
  w.mt = H > 16 ? 2 : 1;
  const int vd = vdim / VG, per = H / VG;
  int worst = 0;
  for (int h0 = 0; h0 < H; h0 += 16 * w.mt) {
    int n = 0;
    for (int m = 0; m < w.mt && h0 + m * 16 < H; ++m) {
      const int a = h0 + m * 16, z = std::min(H, a + 16) - 1;
      n += ((z / per - a / per + 1) * vd + WD_COLS - 1) / WD_COLS;
    }
    worst = std::max(worst, n);
  }
  const int items = (worst + WD_WARPS - 1) / WD_WARPS;
  if (items > 4) return w;
  w.items = items <= 1 ? 1 : (items <= 2 ? 2 : 4);
  auto fits = [&](size_t bytes, int keys, int nbuf) {
    if (bytes > WD_SMEM) return false;
    w.keys = keys; w.nbuf = nbuf; w.smem = bytes;
    return true;
  };
#define WD_TRY(K, N) (w.mt == 2 ? fits(wide_layout<2, K, N>(dim, vdim).total, K, N) : fits(wide_layout<1, K, N>(dim, vdim).total, K, N))
  if (WD_TRY(32, 2) || WD_TRY(16, 2) || WD_TRY(16, 1)) return w;
#undef WD_TRY
  return w;
}

template <typename T, int MT, int KEYS, int NBUF, int ITEMS>
static int wide_launch(const GroupedParams& p, int B, size_t smem, cudaStream_t st) {
  const auto kernel = wide_decode_kernel<T, MT, KEYS, NBUF, ITEMS>;
  cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  kernel<<<dim3(p.splits, (p.H + 16 * MT - 1) / (16 * MT), B), 32 * WD_WARPS, smem, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}
template <typename T, int MT, int KEYS, int NBUF>
static int wide_items(const GroupedParams& p, int B, const WidePlan& w, cudaStream_t st) {
  if (w.items == 1) return wide_launch<T, MT, KEYS, NBUF, 1>(p, B, w.smem, st);
  if (w.items == 2) return wide_launch<T, MT, KEYS, NBUF, 2>(p, B, w.smem, st);
  return wide_launch<T, MT, KEYS, NBUF, 4>(p, B, w.smem, st);
}
template <typename T, int MT>
static int wide_keys(const GroupedParams& p, int B, const WidePlan& w, cudaStream_t st) {
  if (w.keys == 32) return wide_items<T, MT, 32, 2>(p, B, w, st);
  if (w.nbuf == 2) return wide_items<T, MT, 16, 2>(p, B, w, st);
  return wide_items<T, MT, 16, 1>(p, B, w, st);
}

// block = (head, row): merge the slices; exp(sink) joins the denominator (sink null: nothing does)
template <typename T>
__global__ void __launch_bounds__(128) grouped_finish_kernel(const float* __restrict__ ws, const float* __restrict__ stat,
                                                             const T* __restrict__ sink, const T* __restrict__ gate, long long ldg,
                                                             int gate_wide, T* __restrict__ out, int H, int vdim, int ldw, int splits) {
  __shared__ float red[4], fac[GD_MAX_SPLITS];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const long long at = (static_cast<long long>(b) * H + h) * splits;
  const float snk = sink ? Num<T>::to(sink[h]) : -CUDART_INF_F;
  const float m_mine = tid < splits ? stat[(at + tid) * 2] : -CUDART_INF_F;    // splits <= 128: a slice per thread
  float m = fmaxf(m_mine, snk);
#pragma unroll
  for (int off = 16; off > 0; off >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, off));
  if ((tid & 31) == 0) red[tid >> 5] = m;
  __syncthreads();
  m = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
  const float f = m_mine == -CUDART_INF_F ? 0.f : expf(m_mine - m);
  fac[tid] = f;
  const float part = warp_sum(f != 0.f ? stat[(at + tid) * 2 + 1] * f : 0.f);
  __syncthreads();
  if ((tid & 31) == 0) red[tid >> 5] = part;
  __syncthreads();
  const float den = red[0] + red[1] + red[2] + red[3] + (sink ? expf(snk - m) : 0.f);
  const bool narrow = gate != nullptr && !gate_wide;
  const float inv = den > 0.f ? (narrow ? sigmoid_f(Num<T>::to(gate[b * ldg + h])) : 1.0f) / den : 0.f;   // no visible key: zeros
  for (int c = tid; c < vdim; c += blockDim.x) {
    float v = 0.f;
#pragma unroll 8
    for (int s = 0; s < splits; ++s) v = fmaf(ws[(at + s) * ldw + c], fac[s], v);
    if (gate != nullptr && gate_wide) v *= sigmoid_f(Num<T>::to(gate[b * ldg + static_cast<long long>(h) * vdim + c]));
    out[(static_cast<long long>(b) * H + h) * vdim + c] = Num<T>::from(v * inv);
  }
}

static bool gd_use_mma(int dim, int vdim, int dtype) {
  return dtype != OSLO_DT_FP32 && dim % 8 == 0 && vdim % 8 == 0 && dim <= 256 && vdim <= 256;
}

template <typename T, int D>
static int gd_mma_launch(const GroupedParams& p, int B, cudaStream_t st) {
  constexpr size_t smem = gd_mma_smem<D>();
  static_assert(smem >= (GM_HEADS * (D + 8) * 2) + 4 * GM_HEADS * D * sizeof(float), "the stages hold the merge buffer");
  cudaError_t e = cudaFuncSetAttribute(grouped_decode_mma_kernel<T, D>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  const int tiles = (p.H / p.G + GM_HEADS - 1) / GM_HEADS;
  grouped_decode_mma_kernel<T, D><<<dim3(p.splits, p.G * tiles, B), 128, smem, st>>>(p);
  return static_cast<int>(cudaGetLastError());
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
  const size_t a4 = dtype == OSLO_DT_FP32 ? 16 : 8;
  bool vec = dim % 4 == 0 && vdim % 4 == 0 && ldq % 4 == 0 && ldk % 4 == 0 && ldv % 4 == 0;
  for (const void* t : {q, k, v, wq, wk, static_cast<const void*>(q_out), static_cast<const void*>(kc), static_cast<const void*>(vc)})
    vec = vec && aligned_to(t, a4);
  OSLO_DISPATCH_T(dtype, {
    if (vec) qkv_prep_kernel<T, 4><<<static_cast<unsigned>(blocks), 256, 0, stream>>>(p);
    else qkv_prep_kernel<T, 1><<<static_cast<unsigned>(blocks), 256, 0, stream>>>(p);
  });
  return static_cast<int>(cudaGetLastError());
}

extern "C" int oslo_head_prep(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv,
                              const void* wq, const void* wk, float eps, const long long* pos, long long pos_sb, long long pos_ss,
                              const float* freq, int n_freq, int halves, float amplitude, const void* talk, void* q_out, void* kc,
                              long long k_sb, long long k_sg, long long k_st, void* vc, long long v_sb, long long v_sg,
                              long long v_st, const int* lengths, int B, int S, int H, int G, int dim, int vdim, int Tmax,
                              int num_sms, int dtype, int* err_word, cudaStream_t stream) {
  using namespace oslo;
  if (B <= 0 || S <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || dim <= 0 || vdim <= 0 || 2 * n_freq > dim) return -1;
  const long long tokens = static_cast<long long>(B) * S;
  if (tokens > 0x7fffffffll) return -1;
  HeadPrepParams p{q, k, v, ldq, ldk, ldv, wq, wk, pos, pos_sb, pos_ss, freq, n_freq, halves, amplitude, talk, q_out, kc, vc,
                   k_sb, k_sg, k_st, v_sb, v_sg, v_st, lengths, S, H, G, dim, vdim, Tmax, eps, err_word};
  // few tokens: several blocks write the heads of one (each norms all of them first where heads are mixed)
  const int shares = static_cast<int>(std::max<long long>(1, std::min<long long>(talk ? (H + 3) / 4 : (H + HP_WARPS - 1) / HP_WARPS, num_sms / tokens)));
  const int share = (H + shares - 1) / shares;
  const size_t smem = (2 * static_cast<size_t>(n_freq) + 4 + static_cast<size_t>(talk ? H : HP_WARPS) * dim + static_cast<size_t>(HP_WARPS) * dim +
                       (talk ? static_cast<size_t>(share) * H : 0)) * sizeof(float);
  if (smem > 220 * 1024) return -3;
  const size_t a4 = dtype == OSLO_DT_FP32 ? 16 : 8;
  bool vec = dim % 4 == 0 && vdim % 4 == 0;
  for (long long s : {ldq, ldk, ldv, k_sb, k_sg, k_st, v_sb, v_sg, v_st}) vec = vec && s % 4 == 0;
  for (const void* t : {q, k, v, static_cast<const void*>(q_out), static_cast<const void*>(kc), static_cast<const void*>(vc)})
    vec = vec && aligned_to(t, a4);
#define HP_GO(V)                                                                                                               \
  {                                                                                                                            \
    if (smem > 48 * 1024) {                                                                                                    \
      cudaError_t e = cudaFuncSetAttribute(head_prep_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)); \
      if (e != cudaSuccess) return static_cast<int>(e);                                                                        \
    }                                                                                                                          \
    head_prep_kernel<T, V><<<dim3(static_cast<unsigned>(tokens), shares), 32 * HP_WARPS, smem, stream>>>(p);                   \
  }
  OSLO_DISPATCH_T(dtype, { if (vec) HP_GO(4) else HP_GO(1) });
#undef HP_GO
  return static_cast<int>(cudaGetLastError());
}

// whether oslo_grouped_decode runs wide keys (one key head, VG value heads in a cached row) of these sizes
extern "C" int oslo_wide_decode_fits(int H, int VG, int dim, int vdim, int dtype) {
  using namespace oslo;
  if (wide_plan(H, VG, dim, vdim, dtype).keys) return 1;
  const size_t smem = (static_cast<size_t>(GD_HEADS + GD_KEYS) * (dim + 1) + static_cast<size_t>(GD_KEYS) * vdim) * sizeof(float);
  return vdim <= 1024 && smem <= 220 * 1024 ? 1 : 0;
}

extern "C" int oslo_grouped_splits(int B, int H, int G, int VG, int T, int dim, int vdim, int dtype, int num_sms) {
  using namespace oslo;
  const WidePlan wide = VG > 1 ? wide_plan(H, VG, dim, vdim, dtype) : WidePlan{};
  if (wide.keys) {
    // whole waves of blocks: a block costs its share of the keys and some for its start
    const long long blocks = static_cast<long long>(B) * ((H + 16 * wide.mt - 1) / (16 * wide.mt));
    const long long room = static_cast<long long>(num_sms) * std::max<size_t>(1, std::min<size_t>(wide.items > 1 ? 1 : 2, WD_SMEM / (wide.smem + 2048)));
    int best = 1;
    double best_cost = 1e30;
    for (int n = 1; n <= GD_MAX_SPLITS && (n == 1 || n * 64 <= T); ++n) {
      const double cost = static_cast<double>((blocks * n + room - 1) / room) * (static_cast<double>(T) / n + 96.0);
      if (cost < best_cost * 0.999) { best_cost = cost; best = n; }
    }
    return best;
  }
  const int per = gd_use_mma(dim, vdim, dtype) ? GM_HEADS : GD_HEADS;
  const long long blocks = static_cast<long long>(B) * G * ((H / G + per - 1) / per);
  long long s = (3ll * num_sms + blocks - 1) / blocks;
  s = std::min<long long>(s, (T + 127) / 128);           // a slice keeps at least 128 positions of a full cache
  return static_cast<int>(std::max<long long>(1, std::min<long long>(s, GD_MAX_SPLITS)));
}

extern "C" int oslo_grouped_decode(const void* q, const void* kc, const void* vc, const int* lengths, const uint8_t* keep,
                                   long long ld_keep, int n_keep, const void* sink, const void* gate, long long ldg, int gate_wide,
                                   int window, int keep_first, const int* lead, float* ws, float* stat, void* out, int B, int H,
                                   int G, int VG, int dim, int vdim, int Tmax, int splits, float scale, float softcap, int dtype,
                                   int* err_word, cudaStream_t stream) {
  using namespace oslo;
  if (B <= 0 || H <= 0) return 0;
  if (G <= 0 || H % G || B > 65535 || window < 0 || keep_first < 0 || splits < 1 || splits > GD_MAX_SPLITS) return -1;
  if (VG < 1 || (VG > 1 && (G != 1 || H % VG || vdim % VG))) return -1;
  const int vd = vdim / VG;
  GroupedParams p{q, kc, vc, lengths, keep, ld_keep, n_keep, ws, stat, H, G, dim, vdim, (vd + 3) / 4 * 4, Tmax, splits, VG,
                  scale, softcap, window, keep_first, lead, err_word};
#define GD_FINISH(T)                                                                                                               \
  grouped_finish_kernel<T><<<dim3(H, B), 128, 0, stream>>>(ws, stat, static_cast<const T*>(sink), static_cast<const T*>(gate), ldg, \
                                                           gate_wide, static_cast<T*>(out), H, vd, p.ldw, splits)
  const WidePlan wide = VG > 1 && softcap <= 0.f ? wide_plan(H, VG, dim, vdim, dtype) : WidePlan{};
  if (wide.keys && aligned_to(q, 16) && aligned_to(kc, 16) && aligned_to(vc, 16)) {
    int rc = 0;
#define WD_GO(T)                                                                                                       \
  rc = wide.mt == 2 ? wide_keys<T, 2>(p, B, wide, stream) : wide_keys<T, 1>(p, B, wide, stream);                       \
  if (rc == 0) GD_FINISH(T);
    if (dtype == OSLO_DT_BF16) { WD_GO(__nv_bfloat16) } else { WD_GO(__half) }
#undef WD_GO
    return rc ? rc : static_cast<int>(cudaGetLastError());
  }
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
  if (VG == 1 && gd_use_mma(dim, vdim, dtype) && aligned_to(q, 16) && aligned_to(kc, 16) && aligned_to(vc, 16)) {
    const int widest = std::max(dim, vdim);
    int rc = 0;
#define GM_GO(T)                                                                                                              \
  rc = widest <= 64 ? gd_mma_launch<T, 64>(p, B, stream) : (widest <= 128 ? gd_mma_launch<T, 128>(p, B, stream)               \
                                                                           : gd_mma_launch<T, 256>(p, B, stream));            \
  if (rc == 0) GD_FINISH(T);
    if (dtype == OSLO_DT_BF16) { GM_GO(__nv_bfloat16) } else { GM_GO(__half) }
#undef GM_GO
    return rc ? rc : static_cast<int>(cudaGetLastError());
  }
  OSLO_DISPATCH_T(dtype, {
    if (vdim <= 256) GD_GO(1)
    else if (vdim <= 512) GD_GO(2)
    else if (vdim <= 1024) GD_GO(4)
    else return -3;
    GD_FINISH(T);
  });
#undef GD_FINISH
#undef GD_GO
  return static_cast<int>(cudaGetLastError());
}
