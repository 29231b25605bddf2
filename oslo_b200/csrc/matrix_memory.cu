// Matrix memory (mLSTM): gates of a prompt and the decode step. The prompt's recurrence is RULE_MEMORY of linear_recurrence.cu.
//
//   i = cap tanh((z_i + b_i) / cap),  f = log sigmoid(cap tanh((z_f + b_f) / cap)),  m_t = max(f + m_{t-1}, i), m_0 = 0
//   d_t = exp(f + m_{t-1} - m_t),  w_t = exp(i - m_t),  S_t = d_t S_{t-1} + w_t k_t [v_t, 1]^T
//   o_t = S_t^T q_t: the values' columns and, last, n_t . q_t;  y = o / (max(|n_t . q_t|, exp(-m_t)) + 1e-6)
//
// memory_gates_kernel: the maximum is a scan over tokens (F, M): m -> max(F + m, M); a thread composes a stage of 16 tokens, a
// block scans its threads' stages. Within a stage the recurrence keeps its state relative to P, the product of the decays since the
// period's first token, so a token costs two FMAs per state element; a period ends where P would fall below 1e-15, which keeps
// w / P in range whatever the gates are. What is written: P_t (with it the state is read), w_t / P_t, and where a period starts
// what the state has to be multiplied by first (-1: no start). A padded token has d = 1 and w = 0 and never starts a period
// within a stage.
// memory_step_kernel: one token per row. A cluster of blocks per (row, head) shares the value channels; every block computes the
// gates and the normaliser, the norm over the head's outputs is finished over distributed shared memory.
#include <cooperative_groups.h>
#include <math_constants.h>

#include <algorithm>

#include "num.cuh"
#include "oslo_kernels.h"

namespace cg = cooperative_groups;

namespace oslo {

constexpr int MG_STAGE = 16;                // tokens per stage of the recurrence
constexpr float MG_MIN_PERIOD = 1e-15f;
constexpr float MEMORY_FLOOR = 1e-6f;

__device__ __forceinline__ float capped(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

constexpr int MG_SCAN = 128;                                  // threads that scan, a stage each
constexpr int MG_PASS = MG_SCAN * MG_STAGE, MG_PITCH = MG_STAGE + 1;

template <typename T>
__global__ void __launch_bounds__(256) memory_gates_kernel(const float* __restrict__ z, long long ldz, const T* __restrict__ bias,
                                                           float cap, const uint8_t* __restrict__ keep, long long ld_keep,
                                                           float* __restrict__ top, float* __restrict__ read, float* __restrict__ write,
                                                           float* __restrict__ start, float* __restrict__ m_out, int S, int H) {
  __shared__ float warp_f[MG_SCAN / 32], warp_m[MG_SCAN / 32], carry_s;
  // a pass's gates (i, f), then its results (P, w / P, start, m); token t of stage s at s * MG_PITCH + t
  __shared__ float buf[4][MG_SCAN * MG_PITCH];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const float bi = Num<T>::to(bias[h]), bf = Num<T>::to(bias[H + h]);
  float carry = top ? top[static_cast<long long>(b) * H + h] : 0.f;
  const long long at = (static_cast<long long>(b) * H + h) * S, row0 = static_cast<long long>(b) * S;
  for (int base = 0; base < S; base += MG_PASS) {
    const int count = min(MG_PASS, S - base);
#pragma unroll 4
    for (int t = tid; t < MG_PASS; t += 256) {
      float gi = -CUDART_INF_F, gf = 0.f;
      if (t < count && (keep == nullptr || keep[b * ld_keep + base + t])) {
        const float* row = z + (row0 + base + t) * ldz;
        gi = capped(row[h] + bi, cap);
        gf = log_sigmoid(capped(row[H + h] + bf, cap));
      }
      const int o = t / MG_STAGE * MG_PITCH + t % MG_STAGE;
      buf[0][o] = gi;
      buf[1][o] = gf;
    }
    __syncthreads();
    const int o0 = tid * MG_PITCH, n = min(MG_STAGE, count - tid * MG_STAGE);    // n may be <= 0
    float ef = 0.f, em = -CUDART_INF_F;
    if (warp < MG_SCAN / 32) {
      float sf = 0.f, sm = -CUDART_INF_F;
#pragma unroll
      for (int u = 0; u < MG_STAGE; ++u) {
        const float gf = buf[1][o0 + u];
        sf += gf;
        sm = fmaxf(sm + gf, buf[0][o0 + u]);
      }
      // inclusive scan of (F, M) over the warp: first this, then that: (F1 + F2, max(M1 + F2, M2))
#pragma unroll
      for (int off = 1; off < 32; off <<= 1) {
        const float pf = __shfl_up_sync(0xffffffffu, sf, off), pm = __shfl_up_sync(0xffffffffu, sm, off);
        if (lane >= off) { sm = fmaxf(pm + sf, sm); sf += pf; }
      }
      if (lane == 31) { warp_f[warp] = sf; warp_m[warp] = sm; }
      ef = __shfl_up_sync(0xffffffffu, sf, 1);
      em = __shfl_up_sync(0xffffffffu, sm, 1);
    }
    __syncthreads();
    if (warp < MG_SCAN / 32) {
      float m = carry;
      for (int w = 0; w < warp; ++w) m = fmaxf(m + warp_f[w], warp_m[w]);
      if (lane > 0) m = fmaxf(m + ef, em);
      float P = 1.f;
#pragma unroll
      for (int u = 0; u < MG_STAGE; ++u) {
        const float gi = buf[0][o0 + u], gf = buf[1][o0 + u];
        const float top_t = fmaxf(gf + m, gi);
        const float d = expf(gf + m - top_t), w = expf(gi - top_t);
        m = top_t;
        float s = -1.f;
        if (u == 0) {
          s = d;                                 // the kernel multiplies by what the last stage left
        } else if (P * d < MG_MIN_PERIOD) {
          s = P * d;
          P = 1.f;
        } else {
          P *= d;
        }
        buf[0][o0 + u] = P;
        buf[1][o0 + u] = w / P;
        buf[2][o0 + u] = s;
        buf[3][o0 + u] = m;
        if (n > 0 && u == n - 1 && (tid == MG_SCAN - 1 || tid * MG_STAGE + n == count)) carry_s = m;   // the pass's last token
      }
    }
    __syncthreads();
    carry = carry_s;
#pragma unroll 4
    for (int t = tid; t < count; t += 256) {
      const int o = t / MG_STAGE * MG_PITCH + t % MG_STAGE;
      read[at + base + t] = buf[0][o];
      write[at + base + t] = buf[1][o];
      start[at + base + t] = buf[2][o];
      m_out[(row0 + base + t) * H + h] = buf[3][o];
    }
    __syncthreads();
  }
  if (top && tid == 0) top[static_cast<long long>(b) * H + h] = carry;
}

struct MemoryStepParams {
  const void *q, *k, *v, *x, *gate;           // rows b with strides; x: the mixer's input
  long long ldq, ldk, ldv, ldx, ldg;
  const void *w, *bias;                       // [2 H, width], [2 H]: input gates, then forget gates
  const void* norm_w;                         // [H * vdim]
  const uint8_t* keep; long long ld_keep;     // [B, 1], 0 = padding, or nullptr
  float* state;                               // [B, H, dim, lds], column vdim: normaliser
  float* top;                                 // [B, H]
  void* out;                                  // [B, H * vdim]
  int H, dim, vdim, lds, width, cols;         // cols: value channels per CTA
  float cap, q_scale, eps;
};

template <typename T, int VEC, int WV>
__global__ void __launch_bounds__(256) memory_step_kernel(const MemoryStepParams p) {
  extern __shared__ __align__(16) float ms_smem[];
  float* ks = ms_smem;              // [dim], times the write factor
  float* qs = ks + p.dim;           // [dim]
  float* ns = qs + p.dim;           // [dim] normaliser after the token
  float* part = ns + p.dim;         // [ty][cols]
  __shared__ float red[32];
  __shared__ float slice_ss;
  cg::cluster_group cluster = cg::this_cluster();
  const int slices = cluster.num_blocks();
  const int h = blockIdx.y, b = blockIdx.z, c0 = blockIdx.x * p.cols;
  const int cols = max(0, min(p.cols, p.vdim - c0));
  const bool on = p.keep == nullptr || p.keep[b * p.ld_keep];
  const int tx_n = p.cols / VEC;                       // the launcher keeps tx_n <= 256
  const int ty_n = blockDim.x / tx_n;
  const int tx = threadIdx.x % tx_n, ty = threadIdx.x / tx_n;
  float* st0 = p.state + (static_cast<long long>(b) * p.H + h) * p.dim * p.lds;
  float* st = st0 + c0;
  const bool mine = ty < ty_n && tx * VEC < cols;      // VEC > 1: the launcher guarantees vdim % VEC == 0
  constexpr int AHEAD = 4;                             // state rows that are on their way while the gates are computed
  float ahead[AHEAD][VEC];
#pragma unroll
  for (int a = 0; a < AHEAD; ++a)
    if (mine && ty + a * ty_n < p.dim) load_vec<float, VEC>(st + static_cast<long long>(ty + a * ty_n) * p.lds + tx * VEC, ahead[a]);
  const T* q = static_cast<const T*>(p.q) + b * p.ldq + static_cast<long long>(h) * p.dim;
  const T* k = static_cast<const T*>(p.k) + b * p.ldk + static_cast<long long>(h) * p.dim;
  const T* v = static_cast<const T*>(p.v) + b * p.ldv + static_cast<long long>(h) * p.vdim;
  for (int i = threadIdx.x; i < p.dim; i += blockDim.x) ns[i] = st0[static_cast<long long>(i) * p.lds + p.vdim];
  float zi = 0.f, zf = 0.f;
  {
    const T* x = static_cast<const T*>(p.x) + b * p.ldx;
    const T* wi = static_cast<const T*>(p.w) + static_cast<long long>(h) * p.width;
    const T* wf = wi + static_cast<long long>(p.H) * p.width;
    for (int c = threadIdx.x * WV; c < p.width; c += blockDim.x * WV) {
      float xv[WV], a[WV], e[WV];
      load_vec<T, WV>(x + c, xv);
      load_vec<T, WV>(wi + c, a);
      load_vec<T, WV>(wf + c, e);
#pragma unroll
      for (int u = 0; u < WV; ++u) { zi = fmaf(xv[u], a[u], zi); zf = fmaf(xv[u], e[u], zf); }
    }
  }
  zi = block_sum(zi, red);
  zf = block_sum(zf, red);
  const float m_old = p.top[static_cast<long long>(b) * p.H + h];
  float m = m_old, d = 1.f, w = 0.f;
  if (on) {
    const float gi = capped(zi + Num<T>::to(static_cast<const T*>(p.bias)[h]), p.cap);
    const float gf = log_sigmoid(capped(zf + Num<T>::to(static_cast<const T*>(p.bias)[p.H + h]), p.cap));
    m = fmaxf(gf + m_old, gi);
    d = expf(gf + m_old - m);
    w = expf(gi - m);
  }
  float nq = 0.f;
  for (int i = threadIdx.x; i < p.dim; i += blockDim.x) {
    const float kw = Num<T>::to(k[i]) * w, qq = on ? Num<T>::to(q[i]) * p.q_scale : 0.f;
    ks[i] = kw;
    qs[i] = qq;
    const float nn = fmaf(d, ns[i], kw);
    ns[i] = nn;
    nq = fmaf(nn, qq, nq);
  }
  nq = block_sum(nq, red);                             // also makes ks and qs visible
  if (ty < ty_n) {
    const int c = tx * VEC;
    float o[VEC], vv[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      vv[j] = c + j < cols ? Num<T>::to(v[c0 + c + j]) : 0.f;
      o[j] = 0.f;
    }
    auto update = [&](int i, float (&s)[VEC]) {
      const float kk = ks[i], qq = qs[i];
#pragma unroll
      for (int j = 0; j < VEC; ++j) {
        s[j] = fmaf(d, s[j], kk * vv[j]);
        o[j] = fmaf(qq, s[j], o[j]);
      }
      store_vec<float, VEC>(st + static_cast<long long>(i) * p.lds + c, s);
    };
    if (mine) {
#pragma unroll
      for (int a = 0; a < AHEAD; ++a)
        if (ty + a * ty_n < p.dim) update(ty + a * ty_n, ahead[a]);
#pragma unroll 4
      for (int i = ty + AHEAD * ty_n; i < p.dim; i += ty_n) {
        float s[VEC];
        load_vec<float, VEC>(st + static_cast<long long>(i) * p.lds + c, s);
        update(i, s);
      }
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) part[ty * p.cols + c + j] = o[j];
  }
  __syncthreads();
  const float inv = 1.0f / (fmaxf(fabsf(nq), expf(-m)) + MEMORY_FLOOR);
  float ss = 0.f;
  for (int c = threadIdx.x; c < cols; c += blockDim.x) {
    float o = 0.f;
    for (int y = 0; y < ty_n; ++y) o += part[y * p.cols + c];
    o *= inv;
    part[c] = o;                                       // row 0, column c: only this thread reads or writes it now
    ss = fmaf(o, o, ss);
  }
  ss = block_sum(ss, red);
  if (threadIdx.x == 0) slice_ss = ss;
  cluster.sync();                                      // every block has read the old normaliser and maximum by now
  float tot = 0.f;
  for (int r = 0; r < slices; ++r) tot += *cluster.map_shared_rank(&slice_ss, r);
  if (cluster.block_rank() == 0 && on) {
    for (int i = threadIdx.x; i < p.dim; i += blockDim.x) st0[static_cast<long long>(i) * p.lds + p.vdim] = ns[i];
    if (threadIdx.x == 0) p.top[static_cast<long long>(b) * p.H + h] = m;
  }
  cluster.sync();                                      // no CTA leaves while another still reads its shared memory
  const float rn = 1.0f / sqrtf(tot / p.vdim + p.eps);
  T* out = static_cast<T*>(p.out) + (static_cast<long long>(b) * p.H + h) * p.vdim + c0;
  const T* nw = static_cast<const T*>(p.norm_w) + static_cast<long long>(h) * p.vdim + c0;
  const T* gate = static_cast<const T*>(p.gate) + b * p.ldg + static_cast<long long>(h) * p.vdim + c0;
  for (int c = threadIdx.x; c < cols; c += blockDim.x)
    out[c] = Num<T>::from(part[c] * rn * Num<T>::to(nw[c]) * sigmoid_f(Num<T>::to(gate[c])));
}

}  // namespace oslo

extern "C" int oslo_memory_gates(const float* z, long long ldz, const void* bias, float cap, const uint8_t* keep, long long ld_keep,
                                 float* top, float* read, float* write, float* start, float* m_out, int B, int S, int H, int dtype,
                                 cudaStream_t stream) {
  using namespace oslo;
  if (B <= 0 || S <= 0 || H <= 0) return 0;
  if (B > 65535 || !(cap > 0.f)) return -1;
  OSLO_DISPATCH_T(dtype, {
    memory_gates_kernel<T><<<dim3(H, B), 256, 0, stream>>>(z, ldz, static_cast<const T*>(bias), cap, keep, ld_keep, top, read, write,
                                                           start, m_out, S, H);
  });
  return static_cast<int>(cudaGetLastError());
}

extern "C" int oslo_memory_step(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv, const void* x,
                                long long ldx, int width, const void* w, const void* bias, float cap, const void* gate, long long ldg,
                                const void* norm_w, const uint8_t* keep, long long ld_keep, float* state, float* top, void* out,
                                float q_scale, float eps, int B, int H, int dim, int vdim, int num_sms, int dtype, cudaStream_t stream) {
  using namespace oslo;
  if (B <= 0 || H <= 0) return 0;
  if (dim <= 0 || vdim <= 0 || width <= 0 || B > 65535 || H > 65535 || !(cap > 0.f)) return -1;
  MemoryStepParams p{q, k, v, x, gate, ldq, ldk, ldv, ldx, ldg, w, bias, norm_w, keep, ld_keep, state, top, out,
                     H, dim, vdim, (vdim + 1 + 3) / 4 * 4, width, 0, cap, q_scale, eps};
  const int vec = vdim % 4 == 0 && aligned_to(state, 16) ? 4 : 1;
  const size_t te = dtype == OSLO_DT_FP32 ? 4 : 2;
  const bool wide = width % 4 == 0 && ldx % 4 == 0 && aligned_to(x, 4 * te) && aligned_to(w, 4 * te);
  int slices = 1;   // portable cluster sizes; a slice keeps at least 16 columns
  while (slices < 8 && static_cast<long long>(B) * H * slices < 2 * num_sms && vdim / (2 * slices) >= 16) slices *= 2;
  while (slices < 8 && (vdim + slices - 1) / slices > 256 * vec) slices *= 2;
  p.cols = ((vdim + slices - 1) / slices + vec - 1) / vec * vec;
  if (p.cols / vec > 256) return -3;
  const int ty = 256 / (p.cols / vec);
  const size_t smem = (3 * static_cast<size_t>(dim) + static_cast<size_t>(ty) * p.cols) * sizeof(float);
  if (smem > 46 * 1024) return -3;
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
  OSLO_DISPATCH_T(dtype, {
    if (vec == 4) e = wide ? cudaLaunchKernelEx(&cfg, memory_step_kernel<T, 4, 4>, p) : cudaLaunchKernelEx(&cfg, memory_step_kernel<T, 4, 1>, p);
    else e = wide ? cudaLaunchKernelEx(&cfg, memory_step_kernel<T, 1, 4>, p) : cudaLaunchKernelEx(&cfg, memory_step_kernel<T, 1, 1>, p);
  });
  return static_cast<int>(e);
}
