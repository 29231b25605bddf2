// Grouped-query attention with query / key norms, interleaved rotation, capped scores, a sink in the denominator, a window that
// keeps the first keys and an output gate per head:
// what comes before the scores (qkv_prep_kernel) and decoding with one query per row (grouped_decode_kernel). Prompts run
// on the tcgen05 flash kernel (attention_sm100.cu) or, in 32-bit, on sink_attention_kernel (latent_attention.cu).
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

// block = (head, row): merge the slices; exp(sink) joins the denominator (sink null: nothing does)
template <typename T>
__global__ void __launch_bounds__(128) grouped_finish_kernel(const float* __restrict__ ws, const float* __restrict__ stat,
                                                             const T* __restrict__ sink, const T* __restrict__ gate, long long ldg,
                                                             T* __restrict__ out, int H, int vdim, int ldw, int splits) {
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
  const float inv = den > 0.f ? (gate ? sigmoid_f(Num<T>::to(gate[b * ldg + h])) : 1.0f) / den : 0.f;   // no visible key: zeros
  for (int c = tid; c < vdim; c += blockDim.x) {
    float v = 0.f;
#pragma unroll 8
    for (int s = 0; s < splits; ++s) v = fmaf(ws[(at + s) * ldw + c], fac[s], v);
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

extern "C" int oslo_grouped_splits(int B, int H, int G, int T, int dim, int vdim, int dtype, int num_sms) {
  using namespace oslo;
  const int per = gd_use_mma(dim, vdim, dtype) ? GM_HEADS : GD_HEADS;
  const long long blocks = static_cast<long long>(B) * G * ((H / G + per - 1) / per);
  long long s = (3ll * num_sms + blocks - 1) / blocks;
  s = std::min<long long>(s, (T + 127) / 128);           // a slice keeps at least 128 positions of a full cache
  return static_cast<int>(std::max<long long>(1, std::min<long long>(s, GD_MAX_SPLITS)));
}

extern "C" int oslo_grouped_decode(const void* q, const void* kc, const void* vc, const int* lengths, const uint8_t* keep,
                                   long long ld_keep, int n_keep, const void* sink, const void* gate, long long ldg, int window,
                                   int keep_first, const int* lead, float* ws, float* stat, void* out, int B, int H, int G, int dim,
                                   int vdim, int Tmax, int splits, float scale, float softcap, int dtype, int* err_word,
                                   cudaStream_t stream) {
  using namespace oslo;
  if (B <= 0 || H <= 0) return 0;
  if (G <= 0 || H % G || B > 65535 || window < 0 || keep_first < 0 || splits < 1 || splits > GD_MAX_SPLITS) return -1;
  GroupedParams p{q, kc, vc, lengths, keep, ld_keep, n_keep, ws, stat, H, G, dim, vdim, (vdim + 3) / 4 * 4, Tmax, splits,
                  scale, softcap, window, keep_first, lead, err_word};
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
  if (gd_use_mma(dim, vdim, dtype) && aligned_to(q, 16) && aligned_to(kc, 16) && aligned_to(vc, 16)) {
    const int widest = std::max(dim, vdim);
    int rc = 0;
#define GM_GO(T)                                                                                                              \
  rc = widest <= 64 ? gd_mma_launch<T, 64>(p, B, stream) : (widest <= 128 ? gd_mma_launch<T, 128>(p, B, stream)               \
                                                                           : gd_mma_launch<T, 256>(p, B, stream));            \
  if (rc == 0)                                                                                                                \
    grouped_finish_kernel<T><<<dim3(H, B), 128, 0, stream>>>(ws, stat, static_cast<const T*>(sink), static_cast<const T*>(gate), \
                                                             ldg, static_cast<T*>(out), H, vdim, p.ldw, splits);
    if (dtype == OSLO_DT_BF16) { GM_GO(__nv_bfloat16) } else { GM_GO(__half) }
#undef GM_GO
    return rc ? rc : static_cast<int>(cudaGetLastError());
  }
  OSLO_DISPATCH_T(dtype, {
    if (vdim <= 256) GD_GO(1)
    else if (vdim <= 512) GD_GO(2)
    else if (vdim <= 1024) GD_GO(4)
    else return -3;
    grouped_finish_kernel<T><<<dim3(H, B), 128, 0, stream>>>(ws, stat, static_cast<const T*>(sink), static_cast<const T*>(gate), ldg,
                                                             static_cast<T*>(out), H, vdim, p.ldw, splits);
  });
#undef GD_GO
  return static_cast<int>(cudaGetLastError());
}
