// Linear recurrences with a matrix state S (key channels x value channels) per head, in 32-bit floats. Four rules:
//
// RULE_GATED (HGRN2 form): k = (1 - lower) * sigmoid(-(f + f_bias)),  forget gate = 1 - k  (= lower + (1 - lower) * sigmoid(f + f_bias))
//   S_t = S_{t-1} + k_t (v_t - S_{t-1})   per row of the state (a key channel) and column (a value channel)
//   o_t[j] = sum_i silu(q_t)[i] S_t[i, j]
//   `k` is computed from the negated logit, so a gate close to 1 does not lose what it writes to cancellation.
// RULE_DECAY: q, k, v are silu of what is given, S_t = d S_{t-1} + k_t v_t^T with one constant d per head, o_t = S_t^T q_t.
//   Within a period of tokens the state is kept relative to the period's decay: with P_t the product of d over the tokens
//   after the period's first, k_t / P_t is written and P_t q_t reads, which leaves two FMAs per state element and token; the
//   state is multiplied once per period. The period is short enough for 1 / P_t to stay far from overflow, whatever d is.
// RULE_BONUS (RWKV form): decay w_t = exp(-exp(z_t + w0)) per key channel, o_t = S_{t-1}^T r_t + (r_t . (u k_t)) v_t, then
//   S_t = diag(w_t) S_{t-1} + k_t v_t^T.
// RULE_MEMORY (mLSTM form): one decay and one write factor per head and token, S_t = d_t S_{t-1} + w_t k_t [v_t, 1]^T, o_t = S_t^T q_t:
//   the column after the values is the normaliser. Periods as with RULE_DECAY; their starts, P_t and w_t / P_t come from
//   matrix_memory.cu. The first block along the columns also keeps the normaliser, a channel per thread in shared memory: after the
//   conversions of a stage its n . q take two FMAs per channel and token and one reduction over the warp per eight tokens.
//
// Prefill (recurrence_kernel): a thread keeps a 16 x 4 tile of S in registers - rows in pairs, so that every update is a
// packed two-float FMA - and G lanes share a column group; per token it reads 16 + 16 + 4 floats from shared memory,
// does 96 packed FMAs and reduces 4 partial outputs over the G lanes. The prompt is cut into chunks when
// (batch x heads) alone does not fill the GPU: local states of all chunks but the last from zero (no outputs), one
// elementwise scan over the chunks, then every chunk again from its true initial state. Only products of forget gates
// (<= 1) ever appear, so no chunk length can overflow. Three FMAs per state element and token bound the kernel: scalar
// and packed FMAs take the same time here, half the nominal rate, and two resident blocks come close to that.
// Decode (recurrence_step_kernel): a cluster of CTAs per (row, head), each on a slice of the value channels; the RMS
// norm over the head's outputs is finished over distributed shared memory, so a step is one launch.
// Tokens whose `keep` entry is 0 (padding) leave the state as it is and produce zeros.
#include <cooperative_groups.h>

#include <algorithm>

#include "num.cuh"
#include "oslo_kernels.h"

namespace cg = cooperative_groups;

namespace oslo {

enum { RULE_GATED = 0, RULE_DECAY = 1, RULE_BONUS = 2, RULE_MEMORY = 3 };

typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack_f2(float lo, float hi) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ void unpack_f2(f32x2 v, float& lo, float& hi) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
}
__device__ __forceinline__ f32x2 fma_f2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}

__device__ __forceinline__ f32x2 mul_f2(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

// 32-bit models get the accurate exponential; logits that come from 16-bit projections the hardware one (2^-21)
template <typename T> __device__ __forceinline__ float sigmoid_t(float z) {
  return sizeof(T) == 4 ? sigmoid_f(z) : __fdividef(1.0f, 1.0f + __expf(-z));
}
template <typename T> __device__ __forceinline__ float write_gate(float logit, float lower) {
  return (1.0f - lower) * sigmoid_t<T>(-logit);
}
template <typename T> __device__ __forceinline__ float silu_t(float z) { return z * sigmoid_t<T>(z); }
template <typename T> __device__ __forceinline__ float channel_decay(float logit) {
  return sizeof(T) == 4 ? expf(-expf(logit)) : __expf(-__expf(logit));
}

struct RecParams {
  const void *q, *f, *v;             // row (b * S + t) of each has the stride ldq / ldf / ldv; f: gate logits, or the keys
  long long ldq, ldf, ldv;
  const void *f_bias, *lower;        // [H * dim]; RULE_BONUS: w0 and u
  const float* z; long long ldz;     // RULE_BONUS: decay logits [B * S, H * dim]
  const float* head_decay;           // RULE_DECAY: [H]
  const float *read, *write, *start; // RULE_MEMORY: [B, H, S] P_t, w_t / P_t, and what the state is multiplied by where a period starts (< 0: nowhere)
  float q_scale;                     // RULE_MEMORY
  float* norm;                       // RULE_MEMORY: [B, S, H] the normaliser column's outputs
  const uint8_t* keep; long long ld_keep;   // [B, S], 0 = padding, or nullptr
  const float* s_in;                 // initial states, or nullptr (zero)
  float* s_out;                      // final states, or nullptr
  float* decay;                      // STATE_ONLY: product of the forget gates or decays of the chunk
  float* out;                        // [B, S, H, vdim]
  int B, S, H, dim, vdim;
  int lds;                           // elements per state row: vdim; RULE_MEMORY: vdim + 1 and padding, column vdim the normaliser
  int chunk, nchunks;                // tokens per chunk; chunks of this launch per batch row
  float* s_end;                      // last chunk only: final states [B, H, dim, lds], or nullptr
  long long s_batch, s_chunk;        // element strides of s_in / s_out over batch rows and chunks
  int dim_pad;                       // dim rounded up so that every row of a raw stage starts at a 16-byte boundary
  int vec16;                         // q, f, v (and z) rows and head slices start at 16-byte boundaries
};

constexpr int REC_TB = 16;    // tokens staged at a time
constexpr int REC_COLS = 4;   // state columns per thread
constexpr int REC_ROWS = 16;      // state rows per thread

constexpr float REC_MIN_PERIOD = 1e-15f;   // RULE_DECAY: the smallest product of decays within a period

// G lanes per column group. STATE_ONLY: no outputs, start from zero, also the chunk's total decay per row
template <typename T, int G, bool STATE_ONLY, int RULE>
__global__ void __launch_bounds__(RULE == RULE_BONUS ? 128 : 256, RULE == RULE_BONUS ? 3 : 2) recurrence_kernel(const RecParams p) {
  constexpr int DP = REC_ROWS * G;
  constexpr int CONV = DP >= 256 ? 1 : 256 / DP;
  constexpr int PARTS = DP > 32 ? DP / 32 : 1;               // RULE_BONUS: partial sums of r . (u k) per token
  constexpr int WIDTH = G >= REC_COLS ? 1 : REC_COLS / G;    // output columns a lane holds after the reduction
  extern __shared__ float4 rec_smem[];
  const int nt = blockDim.x;
  const int cols = nt / G * REC_COLS;
  float* ks = reinterpret_cast<float*>(rec_smem);
  float* qs = ks + REC_TB * DP;
  float* ws = qs + (STATE_ONLY ? 0 : REC_TB * DP);            // RULE_BONUS: decays
  float* vs = ws + (RULE == RULE_BONUS ? REC_TB * DP : 0);
  __shared__ float bonus_s[RULE == RULE_BONUS && !STATE_ONLY ? REC_TB * PARTS : 1];
  constexpr bool PERIODS = RULE == RULE_DECAY || RULE == RULE_MEMORY;
  __shared__ float read_s[PERIODS ? REC_TB : 1], write_s[PERIODS ? REC_TB : 1];   // P_t, 1 / P_t (RULE_MEMORY: w_t / P_t)
  __shared__ float start_s[RULE == RULE_MEMORY ? 2 * REC_TB : 1], after_s[2];     // [stage parity]: period starts, P of the last token
  __shared__ float n_s[RULE == RULE_MEMORY ? DP : 1], dot_s[RULE == RULE_MEMORY && !STATE_ONLY ? 2 * 8 * REC_TB : 1];   // normaliser; [stage parity][warp][token]
  __shared__ float period_s[RULE == RULE_DECAY ? 2 * REC_TB : 1];   // [stage parity][period]: d^(real tokens - 1), negative: none
  const int tid = threadIdx.x, g = tid % G, cgp = tid / G;
  const int h = blockIdx.y;
  const int b = blockIdx.z / p.nchunks, ch = blockIdx.z % p.nchunks;
  const int col0 = blockIdx.x * cols;
  const int t_begin = ch * p.chunk, t_end = min(p.S, t_begin + p.chunk);
  const T* q = static_cast<const T*>(p.q) + static_cast<long long>(b) * p.S * p.ldq + static_cast<long long>(h) * p.dim;
  const T* f = static_cast<const T*>(p.f) + static_cast<long long>(b) * p.S * p.ldf + static_cast<long long>(h) * p.dim;
  const T* v = static_cast<const T*>(p.v) + static_cast<long long>(b) * p.S * p.ldv + static_cast<long long>(h) * p.vdim + col0;
  const T* fb = static_cast<const T*>(p.f_bias) + h * p.dim;
  const T* lw = static_cast<const T*>(p.lower) + h * p.dim;
  const int my_col = col0 + cgp * REC_COLS;

  // row pair rp of this thread: rows 4 * (g + G * (rp / 2)) + 2 * (rp % 2) and the next one
  f32x2 s[REC_ROWS / 2][REC_COLS];
  const float* sin = p.s_in ? p.s_in + b * p.s_batch + ch * p.s_chunk + static_cast<long long>(h) * p.dim * p.lds : nullptr;
#pragma unroll
  for (int rp = 0; rp < REC_ROWS / 2; ++rp) {
    const int i = 4 * (g + G * (rp / 2)) + 2 * (rp % 2);
#pragma unroll
    for (int c = 0; c < REC_COLS; ++c) {
      float a0 = 0.f, a1 = 0.f;
      if (!STATE_ONLY && sin && my_col + c < p.vdim) {
        if (i < p.dim) a0 = sin[static_cast<long long>(i) * p.lds + my_col + c];
        if (i + 1 < p.dim) a1 = sin[static_cast<long long>(i + 1) * p.lds + my_col + c];
      }
      s[rp][c] = pack_f2(a0, a1);
    }
  }
  float dec[REC_ROWS];
#pragma unroll
  for (int i = 0; i < REC_ROWS; ++i) dec[i] = 1.f;
  const f32x2 minus1 = pack_f2(-1.f, -1.f);
  const float hd = RULE == RULE_DECAY ? p.head_decay[h] : 1.f;
  int period = REC_TB;                                   // RULE_DECAY: tokens between two multiplications of the state
  if (RULE == RULE_DECAY) {
    float least = hd;
    for (int i = 0; i < 4; ++i) least *= least;          // d^16
    while (period > 1 && !(least >= REC_MIN_PERIOD)) {
      period /= 2;
      least = 1.f;
      for (int i = 0; i < period; ++i) least *= hd;
    }
  }
  float pending = 1.f;                                   // what the state still has to be multiplied by
  // where this lane's share of an output row goes, and how many of its WIDTH columns exist (0: another lane writes them)
  int first = 0;
#pragma unroll
  for (int off = G / 2, w = REC_COLS; off > 0 && w > 1; off >>= 1, w /= 2)
    if (g & off) first += w / 2;
  const bool writes = G <= REC_COLS || g % (G / REC_COLS > 0 ? G / REC_COLS : 1) == 0;
  const int out_cols = writes ? min(WIDTH, p.vdim - my_col - first) : 0;
  const long long out_step = static_cast<long long>(p.H) * p.vdim;
  float* out = STATE_ONLY ? nullptr
                          : p.out + ((static_cast<long long>(b) * p.S + t_begin) * p.H + h) * p.vdim + my_col + first;
  // the normaliser: channel i of this head by thread i % blockDim.x; warps without a channel skip it
  const bool has_norm = RULE == RULE_MEMORY && blockIdx.x == 0;
  const int norm_warps = min(nt, DP + 31) / 32;
  float* norm = has_norm && !STATE_ONLY ? p.norm + (static_cast<long long>(b) * p.S + t_begin) * p.H + h : nullptr;
  if (has_norm)
    for (int i = tid; i < DP; i += nt) n_s[i] = !STATE_ONLY && sin && i < p.dim ? sin[static_cast<long long>(i) * p.lds + p.vdim] : 0.f;
  const long long gates_at = RULE == RULE_MEMORY ? (static_cast<long long>(b) * p.H + h) * p.S : 0;

  // raw [REC_TB][raw_ld] stages in the storage type, fetched one step ahead: q (unless STATE_ONLY), f, v slice
  const int f_at = STATE_ONLY ? 0 : p.dim_pad, v_at = f_at + p.dim_pad, raw_ld = v_at + cols;
  float* zraw = vs + REC_TB * cols;                      // RULE_BONUS: [2][REC_TB][dim_pad]
  T* raw = reinterpret_cast<T*>(zraw + (RULE == RULE_BONUS ? 2 * REC_TB * p.dim_pad : 0));
  const float* z = RULE == RULE_BONUS ? p.z + static_cast<long long>(b) * p.S * p.ldz + static_cast<long long>(h) * p.dim : nullptr;
  auto fetch = [&](int t0, int buf) {
    T* dst = raw + static_cast<size_t>(buf) * REC_TB * raw_ld;
    const int n = min(REC_TB, t_end - t0);
    if (RULE == RULE_BONUS) {
      float* zd = zraw + static_cast<size_t>(buf) * REC_TB * p.dim_pad;
      if (p.vec16) {
        const int per = p.dim / 4;
        for (int e = tid; e < n * per; e += nt) {
          const int t = e / per, c = (e - t * per) * 4;
          const uint32_t d32 = static_cast<uint32_t>(__cvta_generic_to_shared(zd + t * p.dim_pad + c));
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d32), "l"(z + (t0 + t) * p.ldz + c) : "memory");
        }
      } else {
        for (int t = 0; t < n; ++t)
          for (int i = tid; i < p.dim; i += nt) zd[t * p.dim_pad + i] = z[(t0 + t) * p.ldz + i];
      }
    }
    if (p.vec16) {
      constexpr int V = 16 / sizeof(T);
      const int per_dim = p.dim / V, per_v = min(cols, p.vdim - col0) / V;
      const int per_row = (STATE_ONLY ? 1 : 2) * per_dim + per_v;
      for (int e = tid; e < n * per_row; e += nt) {
        const int t = e / per_row;
        int c = e - t * per_row;
        const T* src;
        int at;
        if (!STATE_ONLY && c < per_dim) {
          src = q + (t0 + t) * p.ldq + c * V; at = c * V;
        } else {
          if (!STATE_ONLY) c -= per_dim;
          if (c < per_dim) { src = f + (t0 + t) * p.ldf + c * V; at = f_at + c * V; }
          else { c -= per_dim; src = v + (t0 + t) * p.ldv + c * V; at = v_at + c * V; }
        }
        const uint32_t d32 = static_cast<uint32_t>(__cvta_generic_to_shared(dst + t * raw_ld + at));
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d32), "l"(src) : "memory");
      }
    } else {
      const int nv = min(cols, p.vdim - col0);
      for (int t = 0; t < n; ++t) {
        for (int i = tid; i < p.dim; i += nt) {
          if (!STATE_ONLY) dst[t * raw_ld + i] = q[(t0 + t) * p.ldq + i];
          dst[t * raw_ld + f_at + i] = f[(t0 + t) * p.ldf + i];
        }
        for (int c = tid; c < nv; c += nt) dst[t * raw_ld + v_at + c] = v[(t0 + t) * p.ldv + c];
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (t_begin < t_end) fetch(t_begin, 0);
  int it = 0;
  for (int t0 = t_begin; t0 < t_end; t0 += REC_TB, ++it) {
    const int n = min(REC_TB, t_end - t0);
    if (t0 + REC_TB < t_end) {                         // every thread read the other stage before the last barrier
      fetch(t0 + REC_TB, (it + 1) & 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    if (RULE == RULE_DECAY) {                            // read before the second barrier, periods until the stage after next
      for (int s0 = tid * period; s0 < n; s0 += nt * period) {
        float pr = 1.f, ip = 1.f;
        int real = 0;
        const int s1 = min(n, s0 + period);
        for (int t = s0; t < s1; ++t) {
          if (p.keep == nullptr || p.keep[b * p.ld_keep + t0 + t]) {
            if (real++) { pr *= hd; ip = 1.f / pr; }
          }
          read_s[t] = pr;
          write_s[t] = ip;
        }
        period_s[(it & 1) * REC_TB + s0 / period] = real ? pr : -1.f;
      }
    }
    if (RULE == RULE_MEMORY && tid < n) {
      const long long at = gates_at + t0 + tid;
      const float pr = p.read[at];
      read_s[tid] = pr * p.q_scale;
      write_s[tid] = p.write[at];
      start_s[(it & 1) * REC_TB + tid] = p.start[at];
      if (tid == n - 1) after_s[it & 1] = pr;
    }
    __syncthreads();
    const T* src = raw + static_cast<size_t>(it & 1) * REC_TB * raw_ld;
    for (int e = tid; e < DP * CONV; e += nt) {          // CONV threads share a channel's tokens
      const int i = e % DP;
      const bool real = i < p.dim;
      if constexpr (RULE == RULE_GATED) {
        const float bias = real ? Num<T>::to(fb[i]) : 0.f, low = real ? Num<T>::to(lw[i]) : 1.f;
#pragma unroll 4
        for (int t = e / DP; t < n; t += CONV) {
          const bool on = real && (p.keep == nullptr || p.keep[b * p.ld_keep + t0 + t]);
          ks[t * DP + i] = on ? write_gate<T>(Num<T>::to(src[t * raw_ld + f_at + i]) + bias, low) : 0.f;
          if (!STATE_ONLY) qs[t * DP + i] = on ? silu_t<T>(Num<T>::to(src[t * raw_ld + i])) : 0.f;
        }
      } else if constexpr (RULE == RULE_MEMORY) {
#pragma unroll 4
        for (int t = e / DP; t < n; t += CONV) {
          const bool on = real && (p.keep == nullptr || p.keep[b * p.ld_keep + t0 + t]);
          ks[t * DP + i] = on ? Num<T>::to(src[t * raw_ld + f_at + i]) * write_s[t] : 0.f;
          if (!STATE_ONLY) qs[t * DP + i] = on ? Num<T>::to(src[t * raw_ld + i]) * read_s[t] : 0.f;
        }
      } else if constexpr (RULE == RULE_DECAY) {
#pragma unroll 4
        for (int t = e / DP; t < n; t += CONV) {
          const bool on = real && (p.keep == nullptr || p.keep[b * p.ld_keep + t0 + t]);
          ks[t * DP + i] = on ? silu_t<T>(Num<T>::to(src[t * raw_ld + f_at + i])) * write_s[t] : 0.f;
          if (!STATE_ONLY) qs[t * DP + i] = on ? silu_t<T>(Num<T>::to(src[t * raw_ld + i])) * read_s[t] : 0.f;
        }
      } else {
        const float w0 = real ? Num<T>::to(fb[i]) : 0.f, u = real ? Num<T>::to(lw[i]) : 0.f;
        const float* zs = zraw + static_cast<size_t>(it & 1) * REC_TB * p.dim_pad;
        // a warp's threads are at one token (or, with 16 channels, at two); the loop below makes as many turns in each of them
        for (int tt = 0; tt < (REC_TB + CONV - 1) / CONV; ++tt) {
          const int t = e / DP + tt * CONV;
          const bool on = t < n && real && (p.keep == nullptr || p.keep[b * p.ld_keep + t0 + t]);
          const float k = on ? Num<T>::to(src[t * raw_ld + f_at + i]) : 0.f;
          if (t < n) {
            ks[t * DP + i] = k;
            ws[t * DP + i] = on ? channel_decay<T>(zs[t * p.dim_pad + i] + w0) : 1.f;
          }
          if (!STATE_ONLY) {
            const float r = on ? Num<T>::to(src[t * raw_ld + i]) : 0.f;
            if (t < n) qs[t * DP + i] = r;
            float a = r * u * k;
            constexpr int RED = DP < 32 ? DP : 32;
#pragma unroll
            for (int off = RED / 2; off > 0; off >>= 1) a += __shfl_xor_sync(0xffffffffu, a, off);
            if (t < n && i % RED == 0) bonus_s[t * PARTS + i / RED] = a;
          }
        }
      }
    }
    for (int e = tid; e < n * cols; e += nt) {
      const int t = e / cols, c = e - t * cols;
      const float v = col0 + c < p.vdim ? Num<T>::to(src[t * raw_ld + v_at + c]) : 0.f;
      vs[e] = RULE == RULE_DECAY ? silu_t<T>(v) : v;
    }
    if (RULE == RULE_MEMORY && !STATE_ONLY && has_norm && it > 0 && tid < REC_TB) {     // the last stage's n . q
      float a = 0.f;
      for (int w = 0; w < norm_warps; ++w) a += dot_s[((it - 1) & 1) * 8 * REC_TB + w * REC_TB + tid];
      norm[static_cast<long long>((it - 1) * REC_TB + tid) * p.H] = a;
    }
    __syncthreads();
    if (RULE == RULE_MEMORY && has_norm && tid / 32 < norm_warps) {
#pragma unroll 1
      for (int h0 = 0; h0 < n; h0 += 8) {
        float a[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) a[u] = 0.f;
        for (int i = tid; i < DP; i += nt) {
          float nn = n_s[i];
#pragma unroll
          for (int u = 0; u < 8; ++u) {
            const int t = h0 + u;
            if (t < n) {                                 // uniform over the block
              const float f = start_s[(it & 1) * REC_TB + t];
              if (f >= 0.f) nn *= t == 0 ? f * pending : f;
              nn += ks[t * DP + i];
              if (!STATE_ONLY) a[u] = fmaf(nn, qs[t * DP + i], a[u]);
            }
          }
          n_s[i] = nn;
        }
        if (!STATE_ONLY) {                               // eight sums over the warp; lane 4 u ends up with token h0 + u
          const int lane = tid & 31;
#pragma unroll
          for (int off = 16, w = 4; off >= 4; off >>= 1, w >>= 1) {
            const bool upper = (lane & off) != 0;
#pragma unroll
            for (int u = 0; u < 4; ++u) {
              if (u < w) {
                const float mine = upper ? a[u + w] : a[u], give = upper ? a[u] : a[u + w];
                a[u] = mine + __shfl_xor_sync(0xffffffffu, give, off);
              }
            }
          }
          a[0] += __shfl_xor_sync(0xffffffffu, a[0], 2);
          a[0] += __shfl_xor_sync(0xffffffffu, a[0], 1);
          if ((lane & 3) == 0) dot_s[(it & 1) * 8 * REC_TB + tid / 32 * REC_TB + h0 + lane / 4] = a[0];
        }
      }
    }
    for (int t = 0; t < n; ++t) {
      if constexpr (RULE == RULE_MEMORY) {
        float f = start_s[(it & 1) * REC_TB + t];
        if (f >= 0.f) {
          if (t == 0) f *= pending;                      // what the last stage left; within a stage the starts hold it already
          const f32x2 f2 = pack_f2(f, f);
#pragma unroll
          for (int rp = 0; rp < REC_ROWS / 2; ++rp)
#pragma unroll
            for (int c = 0; c < REC_COLS; ++c) s[rp][c] = mul_f2(s[rp][c], f2);
          if (STATE_ONLY) dec[0] *= f;
        }
        if (t == n - 1) pending = after_s[it & 1];
      }
      if (RULE == RULE_DECAY && (t & (period - 1)) == 0) {    // a period begins: its first real token's decay and what is pending
        const float in_period = period_s[(it & 1) * REC_TB + t / period];
        if (in_period >= 0.f) {
          const float f = hd * pending;
          const f32x2 f2 = pack_f2(f, f);
#pragma unroll
          for (int rp = 0; rp < REC_ROWS / 2; ++rp)
#pragma unroll
            for (int c = 0; c < REC_COLS; ++c) s[rp][c] = mul_f2(s[rp][c], f2);
          pending = in_period;
          if (STATE_ONLY) dec[0] *= hd * in_period;
        }
      }
      f32x2 v2[REC_COLS];
      {
        const float4 a = *reinterpret_cast<const float4*>(vs + t * cols + cgp * REC_COLS);
        v2[0] = pack_f2(a.x, a.x); v2[1] = pack_f2(a.y, a.y); v2[2] = pack_f2(a.z, a.z); v2[3] = pack_f2(a.w, a.w);
      }
      f32x2 o2[REC_COLS];
#pragma unroll
      for (int c = 0; c < REC_COLS; ++c) o2[c] = 0ull;
      if (RULE == RULE_BONUS && !STATE_ONLY) {               // this lane's share of (r . (u k)) v
        const f32x2 a2 = g < PARTS ? pack_f2(bonus_s[t * PARTS + g], 0.f) : 0ull;
#pragma unroll
        for (int c = 0; c < REC_COLS; ++c) o2[c] = mul_f2(a2, v2[c]);
      }
#pragma unroll
      for (int kk = 0; kk < REC_ROWS / 4; ++kk) {
        const float4 k4 = *reinterpret_cast<const float4*>(ks + t * DP + 4 * (g + G * kk));
        const f32x2 k2[2] = {pack_f2(k4.x, k4.y), pack_f2(k4.z, k4.w)};
        f32x2 q2[2] = {0ull, 0ull};
        if (!STATE_ONLY) {
          const float4 q4 = *reinterpret_cast<const float4*>(qs + t * DP + 4 * (g + G * kk));
          q2[0] = pack_f2(q4.x, q4.y);
          q2[1] = pack_f2(q4.z, q4.w);
        } else if (RULE == RULE_GATED) {
          dec[4 * kk] *= 1.f - k4.x; dec[4 * kk + 1] *= 1.f - k4.y;
          dec[4 * kk + 2] *= 1.f - k4.z; dec[4 * kk + 3] *= 1.f - k4.w;
        }
        f32x2 w2[2] = {0ull, 0ull};
        if (RULE == RULE_BONUS) {
          const float4 w4 = *reinterpret_cast<const float4*>(ws + t * DP + 4 * (g + G * kk));
          w2[0] = pack_f2(w4.x, w4.y);
          w2[1] = pack_f2(w4.z, w4.w);
          if (STATE_ONLY) { dec[4 * kk] *= w4.x; dec[4 * kk + 1] *= w4.y; dec[4 * kk + 2] *= w4.z; dec[4 * kk + 3] *= w4.w; }
        }
#pragma unroll
        for (int u = 0; u < 2; ++u) {
#pragma unroll
          for (int c = 0; c < REC_COLS; ++c) {
            f32x2& st = s[2 * kk + u][c];
            if (RULE == RULE_GATED) {
              const f32x2 d = fma_f2(st, minus1, v2[c]);
              st = fma_f2(k2[u], d, st);
              if (!STATE_ONLY) o2[c] = fma_f2(q2[u], st, o2[c]);
            } else if (PERIODS) {
              st = fma_f2(k2[u], v2[c], st);
              if (!STATE_ONLY) o2[c] = fma_f2(q2[u], st, o2[c]);
            } else {
              if (!STATE_ONLY) o2[c] = fma_f2(q2[u], st, o2[c]);
              st = fma_f2(w2[u], st, mul_f2(k2[u], v2[c]));
            }
          }
        }
      }
      if (!STATE_ONLY) {
        float o[REC_COLS];
#pragma unroll
        for (int c = 0; c < REC_COLS; ++c) {
          float lo, hi;
          unpack_f2(o2[c], lo, hi);
          o[c] = lo + hi;
        }
        // reduce over the G lanes; each halving step also halves the columns a lane is responsible for
        int width = REC_COLS;
#pragma unroll
        for (int off = G / 2; off > 0; off >>= 1) {
          if (width > 1) {
            const int half = width / 2;
            const bool upper = (g & off) != 0;
#pragma unroll
            for (int c = 0; c < REC_COLS / 2; ++c) {
              if (c < half) {
                const float mine = upper ? o[c + half] : o[c];
                const float give = upper ? o[c] : o[c + half];
                o[c] = mine + __shfl_xor_sync(0xffffffffu, give, off);
              }
            }
            width = half;
          } else {
            o[0] += __shfl_xor_sync(0xffffffffu, o[0], off);
          }
        }
#pragma unroll
        for (int c = 0; c < WIDTH; ++c)
          if (c < out_cols) out[c] = o[c];
        out += out_step;
      }
    }
  }
  if (PERIODS) {
    if (RULE == RULE_MEMORY && STATE_ONLY) dec[0] *= pending;
    const f32x2 f2 = pack_f2(pending, pending);
#pragma unroll
    for (int rp = 0; rp < REC_ROWS / 2; ++rp)
#pragma unroll
      for (int c = 0; c < REC_COLS; ++c) s[rp][c] = mul_f2(s[rp][c], f2);
  }
  if (RULE == RULE_MEMORY && has_norm && !STATE_ONLY) {
    __syncthreads();
    if (it > 0 && tid < REC_TB && t_begin + (it - 1) * REC_TB + tid < t_end) {
      float a = 0.f;
      for (int w = 0; w < norm_warps; ++w) a += dot_s[((it - 1) & 1) * 8 * REC_TB + w * REC_TB + tid];
      norm[static_cast<long long>((it - 1) * REC_TB + tid) * p.H] = a;
    }
  }
  auto store_state = [&](float* so) {
    if (has_norm)
      for (int i = tid; i < p.dim; i += nt) so[static_cast<long long>(i) * p.lds + p.vdim] = n_s[i] * pending;
#pragma unroll
    for (int rp = 0; rp < REC_ROWS / 2; ++rp) {
      const int i = 4 * (g + G * (rp / 2)) + 2 * (rp % 2);
#pragma unroll
      for (int c = 0; c < REC_COLS; ++c) {
        float a0, a1;
        unpack_f2(s[rp][c], a0, a1);
        if (my_col + c < p.vdim) {
          if (i < p.dim) so[static_cast<long long>(i) * p.lds + my_col + c] = a0;
          if (i + 1 < p.dim) so[static_cast<long long>(i + 1) * p.lds + my_col + c] = a1;
        }
      }
    }
  };
  if (p.s_end && ch == p.nchunks - 1) {
    store_state(p.s_end + (static_cast<long long>(b) * p.H + h) * p.dim * p.lds);
  }
  if (p.s_out) {
    store_state(p.s_out + b * p.s_batch + ch * p.s_chunk + static_cast<long long>(h) * p.dim * p.lds);
  }
  if (STATE_ONLY && cgp == 0 && blockIdx.x == 0) {
    float* d = p.decay + ((static_cast<long long>(b) * p.nchunks + ch) * p.H + h) * p.dim;
#pragma unroll
    for (int kk = 0; kk < REC_ROWS / 4; ++kk)
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int i = 4 * (g + G * kk) + u;
        if (i < p.dim) d[i] = PERIODS ? dec[0] : dec[4 * kk + u];
      }
  }
}

// ws[b, c] (c < nchunks - 1) holds the local final state of chunk c; replace every ws[b, c] by the state at the chunk's start
__global__ void __launch_bounds__(256) recurrence_chunk_scan_kernel(float* __restrict__ ws, const float* __restrict__ decay,
                                                                    const float* __restrict__ s_in, int nchunks, int H, int dim,
                                                                    int vdim) {
  const long long per = static_cast<long long>(H) * dim * vdim;
  const long long e = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  const int b = blockIdx.y;
  if (e >= per) return;
  const long long hi = e / vdim;   // head * dim + row
  float s = s_in ? s_in[b * per + e] : 0.f;
#pragma unroll 4
  for (int c = 0; c < nchunks; ++c) {
    const long long o = (static_cast<long long>(b) * nchunks + c) * per + e;
    const bool more = c + 1 < nchunks;
    const float local = more ? ws[o] : 0.f;
    const float d = more ? decay[(static_cast<long long>(b) * (nchunks - 1) + c) * H * dim + hi] : 0.f;
    ws[o] = s;
    s = fmaf(d, s, local);
  }
}

struct StepParams {
  const void *q, *f, *v;
  long long ldq, ldf, ldv;
  const void *f_bias, *lower, *norm_w;      // RULE_BONUS: w0, u, and a norm weight per channel [H * vdim]
  const float* head_decay;                  // RULE_DECAY
  const void* t; long long ldt;             // RULE_BONUS: W_w1 mix [B, rank]
  const void* w2; int rank;                 // ... W_w2 [H * dim, rank]
  const void* gate; long long ldg;          // ... gate logits [B, H * vdim]
  const uint8_t* keep; long long ld_keep;   // [B, 1], 0 = padding, or nullptr
  float* state;      // [B, H, dim, vdim]
  void* out;         // [B, H * vdim]; RULE_DECAY: fp32, not normed
  int H, dim, vdim, cols;   // cols: value channels per CTA
  float eps;
};

template <typename T, int VEC, int RULE>
__global__ void __launch_bounds__(256) recurrence_step_kernel(const StepParams p) {
  extern __shared__ __align__(16) float step_smem[];
  float* ts = step_smem;            // [rank], RULE_BONUS
  float* ks = ts + (RULE == RULE_BONUS ? p.rank : 0);   // [dim]
  float* qs = ks + p.dim;           // [dim]
  float* ws = qs + p.dim;           // [dim], RULE_BONUS
  float* part = ws + (RULE == RULE_BONUS ? p.dim : 0);   // [ty][cols]
  __shared__ float red[32];
  __shared__ float slice_ss;
  cg::cluster_group cluster = cg::this_cluster();
  const int slices = cluster.num_blocks();
  const int h = blockIdx.y, b = blockIdx.z, c0 = blockIdx.x * p.cols;
  const int cols = max(0, min(p.cols, p.vdim - c0));
  const T* q = static_cast<const T*>(p.q) + b * p.ldq + static_cast<long long>(h) * p.dim;
  const T* f = static_cast<const T*>(p.f) + b * p.ldf + static_cast<long long>(h) * p.dim;
  const T* v = static_cast<const T*>(p.v) + b * p.ldv + static_cast<long long>(h) * p.vdim;
  const bool on = p.keep == nullptr || p.keep[b * p.ld_keep];
  const int tx_n = p.cols / VEC;                       // the launcher keeps tx_n <= 256
  const int ty_n = blockDim.x / tx_n;
  const int tx = threadIdx.x % tx_n, ty = threadIdx.x / tx_n;
  float* st = p.state + (static_cast<long long>(b) * p.H + h) * p.dim * p.vdim + c0;
  const bool mine = ty < ty_n && tx * VEC < cols;      // VEC > 1: the launcher guarantees vdim % VEC == 0
  constexpr int AHEAD = 4;                             // state rows that are on their way while the gates are computed
  float ahead[AHEAD][VEC];
#pragma unroll
  for (int a = 0; a < AHEAD; ++a)
    if (mine && ty + a * ty_n < p.dim) load_vec<float, VEC>(st + static_cast<long long>(ty + a * ty_n) * p.vdim + tx * VEC, ahead[a]);
  float bonus = 0.f;
  if constexpr (RULE == RULE_BONUS) {
    const T* t = static_cast<const T*>(p.t) + b * p.ldt;
    for (int i = threadIdx.x; i < p.rank; i += blockDim.x) ts[i] = Num<T>::to(Num<T>::from(tanhf(Num<T>::to(t[i]))));
    __syncthreads();
    const T* w2 = static_cast<const T*>(p.w2) + static_cast<long long>(h) * p.dim * p.rank;
    const T* w0 = static_cast<const T*>(p.f_bias) + h * p.dim;
    int tpr = 1;                                       // threads that share a channel's row of W_w2
    while (tpr < 32 && 2 * tpr * p.dim <= 256) tpr *= 2;
    const int j = threadIdx.x % tpr;
    const bool vec = p.rank % 4 == 0;
    for (int i0 = 0; i0 < p.dim; i0 += 256 / tpr) {    // whole warps stay together
      const int i = i0 + threadIdx.x / tpr;
      float z = 0.f;
      if (i < p.dim) {
        const T* row = w2 + static_cast<long long>(i) * p.rank;
        if (vec) {
#pragma unroll 4
          for (int k = j * 4; k < p.rank; k += 4 * tpr) {
            float w[4];
            load_vec<T, 4>(row + k, w);
            const float4 t4 = *reinterpret_cast<const float4*>(ts + k);
            z = fmaf(w[0], t4.x, fmaf(w[1], t4.y, fmaf(w[2], t4.z, fmaf(w[3], t4.w, z))));
          }
        } else {
          for (int k = j; k < p.rank; k += tpr) z = fmaf(Num<T>::to(row[k]), ts[k], z);
        }
      }
      for (int off = tpr / 2; off > 0; off >>= 1) z += __shfl_xor_sync(0xffffffffu, z, off);
      if (i < p.dim && j == 0) ws[i] = on ? channel_decay<T>(z + Num<T>::to(w0[i])) : 1.f;
    }
    for (int i = threadIdx.x; i < p.dim; i += blockDim.x) {
      ks[i] = on ? Num<T>::to(f[i]) : 0.f;
      qs[i] = on ? Num<T>::to(q[i]) : 0.f;
      bonus = fmaf(qs[i] * Num<T>::to(static_cast<const T*>(p.lower)[h * p.dim + i]), ks[i], bonus);
    }
    bonus = block_sum(bonus, red);
  } else {
    for (int i = threadIdx.x; i < p.dim; i += blockDim.x) {
      if (RULE == RULE_GATED) {
        ks[i] = on ? write_gate<T>(Num<T>::to(f[i]) + Num<T>::to(static_cast<const T*>(p.f_bias)[h * p.dim + i]),
                                Num<T>::to(static_cast<const T*>(p.lower)[h * p.dim + i])) : 0.f;
      } else {
        ks[i] = on ? silu_t<T>(Num<T>::to(f[i])) : 0.f;
      }
      qs[i] = on ? silu_t<T>(Num<T>::to(q[i])) : 0.f;
    }
  }
  __syncthreads();
  const float hd = RULE == RULE_DECAY && on ? p.head_decay[h] : 1.f;
  if (ty < ty_n) {
    const int c = tx * VEC;
    float o[VEC], vv[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      vv[i] = c + i < cols ? Num<T>::to(v[c0 + c + i]) : 0.f;
      if (RULE == RULE_DECAY) vv[i] = silu_t<T>(vv[i]);
      o[i] = RULE == RULE_BONUS && ty == 0 ? bonus * vv[i] : 0.f;
    }
    auto update = [&](int i, float (&s)[VEC]) {
      const float k = ks[i], qq = qs[i], w = RULE == RULE_BONUS ? ws[i] : hd;
#pragma unroll
      for (int j = 0; j < VEC; ++j) {
        if (RULE == RULE_GATED) {
          s[j] = fmaf(k, vv[j] - s[j], s[j]);
          o[j] = fmaf(qq, s[j], o[j]);
        } else if (RULE == RULE_DECAY) {
          s[j] = fmaf(w, s[j], k * vv[j]);
          o[j] = fmaf(qq, s[j], o[j]);
        } else {
          o[j] = fmaf(qq, s[j], o[j]);
          s[j] = fmaf(w, s[j], k * vv[j]);
        }
      }
      store_vec<float, VEC>(st + static_cast<long long>(i) * p.vdim + c, s);
    };
    if (mine) {
#pragma unroll
      for (int a = 0; a < AHEAD; ++a)
        if (ty + a * ty_n < p.dim) update(ty + a * ty_n, ahead[a]);
#pragma unroll 4
      for (int i = ty + AHEAD * ty_n; i < p.dim; i += ty_n) {
        float s[VEC];
        load_vec<float, VEC>(st + static_cast<long long>(i) * p.vdim + c, s);
        update(i, s);
      }
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) part[ty * p.cols + c + j] = o[j];
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = threadIdx.x; c < cols; c += blockDim.x) {
    float o = 0.f;
    for (int y = 0; y < ty_n; ++y) o += part[y * p.cols + c];
    part[c] = o;                                       // row 0, column c: only this thread reads or writes it now
    ss = fmaf(o, o, ss);
    if (RULE == RULE_DECAY) static_cast<float*>(p.out)[(static_cast<long long>(b) * p.H + h) * p.vdim + c0 + c] = o;
  }
  if (RULE == RULE_DECAY) return;                      // the norm runs over all heads
  ss = block_sum(ss, red);
  if (threadIdx.x == 0) slice_ss = ss;
  cluster.sync();
  float tot = 0.f;
  for (int r = 0; r < slices; ++r) tot += *cluster.map_shared_rank(&slice_ss, r);
  cluster.sync();                                      // no CTA leaves while another still reads its shared memory
  const float rn = 1.0f / sqrtf(tot / p.vdim + p.eps);
  T* out = static_cast<T*>(p.out) + (static_cast<long long>(b) * p.H + h) * p.vdim + c0;
  const T* nw = static_cast<const T*>(p.norm_w) + (RULE == RULE_BONUS ? static_cast<long long>(h) * p.vdim : 0) + c0;
  const T* gate = RULE == RULE_BONUS ? static_cast<const T*>(p.gate) + b * p.ldg + static_cast<long long>(h) * p.vdim + c0 : nullptr;
  for (int c = threadIdx.x; c < cols; c += blockDim.x) {
    float y = part[c] * rn * Num<T>::to(nw[c]);
    if (RULE == RULE_BONUS) y *= silu_t<T>(Num<T>::to(gate[c]));
    out[c] = Num<T>::from(y);
  }
}

// threads of a block: the column groups of a head, at most 256 (128 with the bonus rule, whose decays need more registers)
static int rec_threads(int g, int vdim, int rule) {
  const int groups = (vdim + REC_COLS - 1) / REC_COLS;
  return std::min(rule == RULE_BONUS ? 128 : 256, (groups * g + 31) / 32 * 32);
}

template <typename T, int G, bool STATE_ONLY, int RULE>
static int rec_launch(const RecParams& p, cudaStream_t st) {
  const int nt = rec_threads(G, p.vdim, RULE), cols = nt / G * REC_COLS;
  const int rows = (STATE_ONLY ? 1 : 2) + (RULE == RULE_BONUS ? 1 : 0);
  const size_t smem = static_cast<size_t>(REC_TB) * ((rows * REC_ROWS * G + cols + (RULE == RULE_BONUS ? 2 * p.dim_pad : 0)) * sizeof(float) +
                                                     2 * ((STATE_ONLY ? 1 : 2) * p.dim_pad + cols) * sizeof(T));
  if (smem > 44 * 1024) {      // static arrays come on top
    cudaError_t e = cudaFuncSetAttribute(recurrence_kernel<T, G, STATE_ONLY, RULE>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  dim3 grid((p.vdim + cols - 1) / cols, p.H, p.B * p.nchunks);
  recurrence_kernel<T, G, STATE_ONLY, RULE><<<grid, nt, smem, st>>>(p);
  return static_cast<int>(cudaGetLastError());
}
template <typename T, bool STATE_ONLY, int RULE>
static int rec_dispatch_rule(const RecParams& p, cudaStream_t st) {
  if (p.dim <= 16) return rec_launch<T, 1, STATE_ONLY, RULE>(p, st);
  if (p.dim <= 32) return rec_launch<T, 2, STATE_ONLY, RULE>(p, st);
  if (p.dim <= 64) return rec_launch<T, 4, STATE_ONLY, RULE>(p, st);
  if (p.dim <= 128) return rec_launch<T, 8, STATE_ONLY, RULE>(p, st);
  if (p.dim <= 256) return rec_launch<T, 16, STATE_ONLY, RULE>(p, st);
  if constexpr (RULE != RULE_BONUS)                     // the bonus rule's stages of 512 channels exceed the shared memory
    if (p.dim <= 512) return rec_launch<T, 32, STATE_ONLY, RULE>(p, st);
  return -3;
}
template <typename T, bool STATE_ONLY>
static int rec_dispatch(const RecParams& p, int rule, cudaStream_t st) {
  if (rule == RULE_GATED) return rec_dispatch_rule<T, STATE_ONLY, RULE_GATED>(p, st);
  if (rule == RULE_DECAY) return rec_dispatch_rule<T, STATE_ONLY, RULE_DECAY>(p, st);
  if (rule == RULE_BONUS) return rec_dispatch_rule<T, STATE_ONLY, RULE_BONUS>(p, st);
  if (rule == RULE_MEMORY) return rec_dispatch_rule<T, STATE_ONLY, RULE_MEMORY>(p, st);
  return -1;
}

}  // namespace oslo

// how many chunks a prompt of S tokens is cut into so that the recurrence fills the GPU
extern "C" int oslo_recurrence_chunks(int rule, int B, int S, int H, int dim, int vdim, int num_sms) {
  using namespace oslo;
  int g = 1;
  while (REC_ROWS * g < dim && g < 32) g *= 2;
  const int nt = rec_threads(g, vdim, rule), cols = nt / g * REC_COLS;
  const long long ctas = static_cast<long long>(B) * H * ((vdim + cols - 1) / cols);
  if (S < 128) return 1;
  // an SM's blocks share its FMA pipes: time ~ (blocks of the fullest SM) x (tokens per chunk); more than one chunk adds the
  // local states (two thirds of the work, all chunks but the last) and the scan
  int best = 1;
  double best_cost = 1e30;
  for (int n = 1; n <= S / 64 && n <= 64; ++n) {
    const double per = static_cast<double>(S) / n;
    // the fullest SM runs its blocks in waves of as many as fit; in units of 256 threads, of which too few leave its pipes partly idle
    const int fit = std::max(1, (rule == RULE_BONUS ? 384 : 512) / nt);
    const auto time = [&](long long blocks) {
      const int most = static_cast<int>((blocks + num_sms - 1) / num_sms), waves = most / fit, rest = most % fit;
      const double unit = nt / 256.0;
      return waves * fit * unit + (rest ? std::max(waves ? 1.0 : 1.4, rest * unit) : 0.0);
    };
    const double c3 = time(ctas * n) * per;
    // ... and the states' four trips through memory (16 bytes per element, in units of one token's update)
    const double c1 = n > 1 ? time(ctas * (n - 1)) * per * 0.67 + 40.0 + 0.094 * B * H * n : 0.0;
    if (c3 + c1 < best_cost) { best_cost = c3 + c1; best = n; }
  }
  return best;
}

static int run_recurrence(int rule, oslo::RecParams& p, float* state, float* ws, float* decay, int nchunks, int dtype,
                          cudaStream_t stream) {
  using namespace oslo;
  const int B = p.B, S = p.S, H = p.H, dim = p.dim, vdim = p.vdim;
  if (B <= 0 || S <= 0 || H <= 0) return 0;
  if (dim <= 0 || vdim <= 0 || dim > 512 || H > 65535 || nchunks < 1 || static_cast<long long>(B) * nchunks > 65535) return -1;
  p.lds = rule == RULE_MEMORY ? (vdim + 1 + 3) / 4 * 4 : vdim;
  const long long per = static_cast<long long>(H) * dim * p.lds;
  const int te = dtype == OSLO_DT_FP32 ? 4 : 2, v16 = 16 / te;
  p.dim_pad = (dim + 7) / 8 * 8;
  p.vec16 = dim % v16 == 0 && vdim % v16 == 0 && p.ldq % v16 == 0 && p.ldf % v16 == 0 && p.ldv % v16 == 0 && aligned_to(p.q, 16) &&
            aligned_to(p.f, 16) && aligned_to(p.v, 16) && (rule != RULE_BONUS || (p.ldz % 4 == 0 && aligned_to(p.z, 16)));
  int rc = 0;
  if (nchunks == 1) {
    p.chunk = S; p.nchunks = 1; p.s_in = state; p.s_out = state; p.s_batch = per; p.s_chunk = 0;
    OSLO_DISPATCH_T(dtype, { rc = rec_dispatch<T, false>(p, rule, stream); });
    return rc;
  }
  if (ws == nullptr || decay == nullptr) return -1;
  p.nchunks = nchunks;
  p.chunk = ((S + nchunks - 1) / nchunks + REC_TB - 1) / REC_TB * REC_TB;
  p.s_batch = per * nchunks; p.s_chunk = per;
  p.s_in = nullptr; p.s_out = ws; p.decay = decay;
  p.nchunks = nchunks - 1;             // nobody starts from the last chunk's state
  OSLO_DISPATCH_T(dtype, { rc = rec_dispatch<T, true>(p, rule, stream); });
  if (rc) return rc;
  recurrence_chunk_scan_kernel<<<dim3(static_cast<unsigned>((per + 255) / 256), B), 256, 0, stream>>>(ws, decay, state, nchunks, H,
                                                                                                     dim, p.lds);
  rc = static_cast<int>(cudaGetLastError());
  if (rc) return rc;
  p.nchunks = nchunks;
  p.s_in = ws; p.s_out = nullptr; p.s_end = state;
  OSLO_DISPATCH_T(dtype, { rc = rec_dispatch<T, false>(p, rule, stream); });
  return rc;
}

// f_bias / lower: the gate bias and lower bound (RULE_GATED), or w0 and u (RULE_BONUS); z: decay logits (RULE_BONUS);
// head_decay: RULE_DECAY
extern "C" int oslo_recurrence(int rule, const void* q, long long ldq, const void* f, long long ldf, const void* v, long long ldv,
                               const void* f_bias, const void* lower, const float* z, long long ldz, const float* head_decay,
                               const uint8_t* keep, long long ld_keep, float* state, float* out, float* ws, float* decay, int nchunks,
                               int B, int S, int H, int dim, int vdim, int dtype, cudaStream_t stream) {
  oslo::RecParams p{};
  if (rule == oslo::RULE_MEMORY) return -1;
  p.q = q; p.f = f; p.v = v; p.ldq = ldq; p.ldf = ldf; p.ldv = ldv; p.f_bias = f_bias; p.lower = lower;
  p.z = z; p.ldz = ldz; p.head_decay = head_decay;
  p.keep = keep; p.ld_keep = ld_keep; p.out = out;
  p.B = B; p.S = S; p.H = H; p.dim = dim; p.vdim = vdim;
  return run_recurrence(rule, p, state, ws, decay, nchunks, dtype, stream);
}

extern "C" int oslo_memory_recurrence(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv,
                                      const float* read, const float* write, const float* start, float q_scale, const uint8_t* keep,
                                      long long ld_keep, float* state, float* out, float* norm, float* ws, float* decay, int nchunks,
                                      int B, int S, int H, int dim, int vdim, int dtype, cudaStream_t stream) {
  oslo::RecParams p{};
  p.q = q; p.f = k; p.v = v; p.ldq = ldq; p.ldf = ldk; p.ldv = ldv; p.read = read; p.write = write; p.start = start; p.q_scale = q_scale;
  p.keep = keep; p.ld_keep = ld_keep; p.out = out; p.norm = norm;
  p.B = B; p.S = S; p.H = H; p.dim = dim; p.vdim = vdim;
  return run_recurrence(oslo::RULE_MEMORY, p, state, ws, decay, nchunks, dtype, stream);
}

static int step_launch(int rule, oslo::StepParams p, int B, int num_sms, int dtype, cudaStream_t stream) {
  using namespace oslo;
  if (B <= 0 || p.H <= 0) return 0;
  if (p.dim <= 0 || p.vdim <= 0 || B > 65535 || p.H > 65535) return -1;
  const int H = p.H, vdim = p.vdim;
  const int vec = vdim % 4 == 0 && aligned_to(p.state, 16) ? 4 : 1;
  int slices = 1;   // portable cluster sizes; a slice keeps at least 16 columns
  while (slices < 8 && static_cast<long long>(B) * H * slices < 2 * num_sms && vdim / (2 * slices) >= 16) slices *= 2;
  while (slices < 8 && (vdim + slices - 1) / slices > 256 * vec) slices *= 2;
  p.cols = ((vdim + slices - 1) / slices + vec - 1) / vec * vec;
  if (p.cols / vec > 256) return -3;
  const int ty = 256 / (p.cols / vec);
  const size_t smem = ((rule == RULE_BONUS ? 3 : 2) * static_cast<size_t>(p.dim) + p.rank + static_cast<size_t>(ty) * p.cols) * sizeof(float);
  if (smem > 48 * 1024) return -3;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(slices, H, B);
  cfg.blockDim = dim3(256);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = slices; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  cudaError_t e = cudaSuccess;
#define STEP_GO(R)                                                                    \
  if (vec == 4) e = cudaLaunchKernelEx(&cfg, recurrence_step_kernel<T, 4, R>, p);     \
  else e = cudaLaunchKernelEx(&cfg, recurrence_step_kernel<T, 1, R>, p);
  OSLO_DISPATCH_T(dtype, {
    if (rule == RULE_GATED) { STEP_GO(RULE_GATED) }
    else if (rule == RULE_DECAY) { STEP_GO(RULE_DECAY) }
    else { STEP_GO(RULE_BONUS) }
  });
#undef STEP_GO
  return static_cast<int>(e);
}

extern "C" int oslo_recurrence_step(const void* q, long long ldq, const void* f, long long ldf, const void* v, long long ldv,
                                    const void* f_bias, const void* lower, const void* norm_w, const uint8_t* keep,
                                    long long ld_keep, float* state, void* out, float eps, int B, int H, int dim, int vdim, int num_sms, int dtype, cudaStream_t stream) {
  oslo::StepParams p{};
  p.q = q; p.f = f; p.v = v; p.ldq = ldq; p.ldf = ldf; p.ldv = ldv;
  p.f_bias = f_bias; p.lower = lower; p.norm_w = norm_w; p.keep = keep; p.ld_keep = ld_keep;
  p.state = state; p.out = out; p.H = H; p.dim = dim; p.vdim = vdim; p.eps = eps;
  return step_launch(oslo::RULE_GATED, p, B, num_sms, dtype, stream);
}

extern "C" int oslo_decayed_step(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv,
                                 const float* head_decay, const uint8_t* keep, long long ld_keep, float* state, float* out, int B,
                                 int H, int dim, int vdim, int num_sms, int dtype, cudaStream_t stream) {
  oslo::StepParams p{};
  p.q = q; p.f = k; p.v = v; p.ldq = ldq; p.ldf = ldk; p.ldv = ldv; p.head_decay = head_decay; p.keep = keep; p.ld_keep = ld_keep;
  p.state = state; p.out = out; p.H = H; p.dim = dim; p.vdim = vdim;
  return step_launch(oslo::RULE_DECAY, p, B, num_sms, dtype, stream);
}

extern "C" int oslo_bonus_step(const void* r, long long ldr, const void* k, long long ldk, const void* v, long long ldv, const void* t,
                               long long ldt, const void* w2, int rank, const void* w0, const void* u, const void* norm_w,
                               const void* gate, long long ldg, const uint8_t* keep, long long ld_keep, float* state, void* out,
                               float eps, int B, int H, int dim, int vdim, int num_sms, int dtype, cudaStream_t stream) {
  oslo::StepParams p{};
  p.q = r; p.f = k; p.v = v; p.ldq = ldr; p.ldf = ldk; p.ldv = ldv; p.f_bias = w0; p.lower = u; p.norm_w = norm_w;
  p.t = t; p.ldt = ldt; p.w2 = w2; p.rank = rank; p.gate = gate; p.ldg = ldg;
  p.keep = keep; p.ld_keep = ld_keep; p.state = state; p.out = out; p.H = H; p.dim = dim; p.vdim = vdim; p.eps = eps;
  return step_launch(oslo::RULE_BONUS, p, B, num_sms, dtype, stream);
}
