// Flash attention on the 5th-generation tensor cores (tcgen05 + TMEM), forward pass.
//
// One CTA owns 128 query rows of one (batch, head); one TMEM lane per row. 192 threads:
//   warp 0     TMA producer: Q once, then K and V blocks through two 2-deep shared-memory rings
//   warp 1     TMEM owner + the single MMA-issuing lane
//   warps 2-5  softmax: thread = query row. They read S = Q K^T from TMEM (tcgen05.ld), apply the mask
//              (causal with query offset, sliding window, key padding), keep the running max / sum, write
//              P = exp2(S - m) as 16-bit pairs back into the TMEM columns S came from (the next MMA reads its A
//              operand from tensor memory; a shared-memory P tile in the 128-byte-swizzled K-major layout is
//              the alternative path), and rescale the O accumulator in TMEM only when the running max has grown
//              by more than 2^8 (warp-uniform decision), so most blocks never touch O.
// S is double-buffered in TMEM so Q K^T of block j+1 runs under the softmax of block j, and P V of block j runs
// under the softmax of block j+1. O (128 x D fp32) stays in TMEM for the whole row of blocks.
// The K tile [BN x 64]-column sub-tiles are at the same time the MN-major image of V that P V needs, so K and V
// use the same TMA box and no transposes exist anywhere. Every wait is bounded (ptx.cuh).
//
// Reference behaviour covered: the materialised-score path Q K^T -> scaled (upper-triangular | padding) masked
// softmax -> P V of oslo/models/gptj/modeling_gptj.py:151-191 with the kernels of
// oslo/fused_kernels/includes/fused_triang_softmax.h:134-351 and fused_softmax.h:111-325 (sequence length <= 2048
// there; no limit here), plus GPT-Neo's local window (oslo/models/gpt_neo/modeling_gpt_neo.py:150-160).
#include "attention_sm100.cuh"

namespace oslo {

constexpr float FA_RESCALE_THRESHOLD = 8.0f;  // log2 units

struct FaParams {
  void* out;          // [B, H, Sq, D] element strides below
  float* lse;         // [B, H, Sq]
  const uint8_t* kpm; // [B, Sk] 1 = keep, or nullptr
  int B, H, Sq, Sk;
  long long o_sb, o_sh, o_ss;
  float scale;
  int causal, window;
  int fp16;
  // position of the (seq, head, batch) coordinates inside each 4-D tensor map (dim 0 is always D)
  int q_pos[3], k_pos[3], v_pos[3];
  int* err;
  int group;            // query heads per key / value head
  float softcap;        // CAP kernels: scores become softcap * tanh(score / softcap)
  // softmax with a sink and an output gate (null: without): exp(sink[h]) joins the denominator, row s of
  // head h is multiplied by sigmoid(gate[(b * Sq + s) * ldg + h]), or (gate_wide) every element by that of
  // gate[(b * Sq + s) * ldg + h * d_out + column]; only the first d_out columns are stored
  const void* sink;
  const void* gate;
  long long ldg;
  int d_out, gate_wide;
  // a window that also sees the sequence's first keep_first keys; lead [B] (or nullptr): padding ahead of a sequence
  int keep_first;
  const int* lead;
  // 64-column sub-tiles of the query and key operands that come from tq / tk; the others come from tq2 / tk2 (a part
  // of the keys that all heads share)
  int sub_first;
  int q2_pos[3], k2_pos[3];
};

// Which blocks of BN keys the 128 query rows from q0 on read: the kept keys' blocks ahead of the window's come first
struct FaBlocks {
  int offset, lead, kept_lo, key_lo, nkept, n, bn;
  __device__ __forceinline__ FaBlocks(const FaParams& p, int b, int q0, int BN) {
    bn = BN;
    offset = p.Sk - p.Sq;
    int key_hi = p.Sk;
    key_lo = 0;
    if (p.causal) key_hi = min(p.Sk, q0 + FA_BM + offset);
    if (p.window > 0) key_lo = max(0, q0 + offset - p.window + 1) / BN * BN;
    lead = p.lead ? p.lead[b] : 0;
    kept_lo = max(0, lead) / BN * BN;
    const int kept_hi = min(key_lo, lead + p.keep_first);
    nkept = kept_hi > kept_lo ? (kept_hi - kept_lo + BN - 1) / BN : 0;
    n = nkept + (key_hi > key_lo ? (key_hi - key_lo + BN - 1) / BN : 0);
  }
  __device__ __forceinline__ int start(int j) const { return j < nkept ? kept_lo + j * bn : key_lo + (j - nkept) * bn; }
};

// The four softmax warps of both kernels: S from TMEM columns [0, BN) and [BN, 2 BN), O (D columns) from 2 BN on. Barriers by
// number from bar0: 0 q_full, then (second phase) the last P V is done | 9,10 s_full | 11,12 s_empty | 13 p_ready[0] | 14 pv_done | 15 p_ready[1] (PT only: one per S/P buffer)
template <int BN, bool PT, bool CAP>
__device__ __forceinline__ void fa_softmax_warps(const FaParams& p, const int D, const FaBlocks& blocks, uint32_t tmem_base, uint32_t bar0,
                                                 uint32_t p_s, volatile int* abort_flag, int warp, int lane, int b, int h, int q0) {
  constexpr uint32_t Q_SUB = FA_BM * 128, O_COL = 2 * BN;
  auto bar = [&](int i) { return bar0 + 8u * i; };
  const int offset = blocks.offset;
  const int quad = warp & 3;
  const int row_l = quad * 32 + lane;
  const int row = q0 + row_l;
  const uint32_t t_lane = tmem_base + (static_cast<uint32_t>(quad * 32) << 16);
  const uint8_t* kpm_row = p.kpm ? p.kpm + static_cast<long long>(b) * p.Sk : nullptr;
  const float sc = CAP ? 2.f * FA_LOG2E * p.scale / p.softcap : p.scale * FA_LOG2E;
  const float cap = p.softcap * FA_LOG2E;
  const bool fp16 = p.fp16 != 0;
  float m_ref = -CUDART_INF_F, l_sum = 0.f;
  bool ok = true;
  for (int j = 0; j < blocks.n && ok; ++j) {
    const int st = j & 1;
    const int n0 = blocks.start(j);
    ok = mbar_wait_warp(bar(9 + st), (j >> 1) & 1, abort_flag, p.err, ERR_WAIT_TMEM_FULL);
    if (!ok) break;
    tc_fence_after();
    float s[BN];
#pragma unroll
    for (int c0 = 0; c0 < BN; c0 += 32) {
      uint32_t r[32];
      tmem_ld_32x32(t_lane + st * BN + c0, r);
      tmem_wait_ld();
#pragma unroll
      for (int i = 0; i < 32; ++i) {
        s[c0 + i] = __uint_as_float(r[i]) * sc;
        if (CAP) s[c0 + i] = cap - __fdividef(2.f * cap, exp2f(s[c0 + i]) + 1.f);
      }
    }
    tc_fence_before();
    __syncwarp();
    if (lane == 0) mbar_arrive(bar(11 + st));  // S buffer may be overwritten by Q K^T of block j + 2
    // ---- mask (only blocks that touch the diagonal, the window edge, the end of the keys, or padding)
    const bool need_mask = (n0 + BN > p.Sk) || kpm_row != nullptr ||
                           (p.causal && n0 + BN - 1 > q0 + offset) ||
                           (p.window > 0 && n0 <= q0 + FA_BM - 1 + offset - p.window);
    if (need_mask) {
      // one bit per column: up to `last`, and from `first` on or before `kept`
      const int qpos = row + offset;
      const int last = p.causal ? min(p.Sk - 1, qpos) : p.Sk - 1;
      const int first = p.window > 0 ? qpos - p.window + 1 : 0, kept = p.window > 0 ? blocks.lead + p.keep_first : 0;
      auto below = [](int n) { return n <= 0 ? 0u : (n >= 32 ? 0xffffffffu : (1u << n) - 1u); };
#pragma unroll
      for (int c0 = 0; c0 < BN; c0 += 32) {
        const int base = n0 + c0;
        uint32_t vis = below(last - base + 1) & (~below(first - base) | below(kept - base));
        if (kpm_row) vis &= __ballot_sync(0xffffffffu, base + lane < p.Sk && kpm_row[base + lane] != 0);
#pragma unroll
        for (int i = 0; i < 32; ++i)
          if (!((vis >> i) & 1u)) s[c0 + i] = -CUDART_INF_F;
      }
    }
    // four independent chains: one thread per row means nothing else hides the latency of a 64-long dependent chain
    float mx4[4] = {s[0], s[1], s[2], s[3]};
#pragma unroll
    for (int i = 4; i < BN; i += 4) {
      mx4[0] = fmaxf(mx4[0], s[i]);
      mx4[1] = fmaxf(mx4[1], s[i + 1]);
      mx4[2] = fmaxf(mx4[2], s[i + 2]);
      mx4[3] = fmaxf(mx4[3], s[i + 3]);
    }
    const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
    const float m_new = fmaxf(m_ref, mx);
    // rescale O only when some row of this warp outgrew its reference by 2^8 (or on the first block)
    const bool grow = (j == 0) || (m_new - m_ref > FA_RESCALE_THRESHOLD);
    const bool rescale = __any_sync(0xffffffffu, grow);
    float factor = 1.f;
    if (rescale) {
      factor = (m_ref == -CUDART_INF_F) ? 0.f : exp2f(m_ref - m_new);
      m_ref = m_new;
      l_sum *= factor;
    }
    const float m_use = (m_ref == -CUDART_INF_F) ? 0.f : m_ref;
    float ps4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int i = 0; i < BN; i += 4) {
      s[i] = exp2f(s[i] - m_use);
      s[i + 1] = exp2f(s[i + 1] - m_use);
      s[i + 2] = exp2f(s[i + 2] - m_use);
      s[i + 3] = exp2f(s[i + 3] - m_use);
      ps4[0] += s[i];
      ps4[1] += s[i + 1];
      ps4[2] += s[i + 2];
      ps4[3] += s[i + 3];
    }
    l_sum += (ps4[0] + ps4[1]) + (ps4[2] + ps4[3]);
    // the shared P tile is single-buffered, so P V of block j-1 must have finished before it is rewritten; the
    // TMEM P buffers alternate, so there only a rescale of O has to wait for it
    if (j > 0 && (!PT || rescale)) {
      ok = mbar_wait_warp(bar(14), (j - 1) & 1, abort_flag, p.err, ERR_WAIT_TMEM_FULL);
      if (!ok) break;
      tc_fence_after();
      if (rescale) {
#pragma unroll 1
        for (int c0 = 0; c0 < D; c0 += 32) {
          uint32_t r[32];
          tmem_ld_32x32(t_lane + O_COL + c0, r);
          tmem_wait_ld();
#pragma unroll
          for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * factor);
          tmem_st_32x32(t_lane + O_COL + c0, r);
        }
        tmem_wait_st();
      }
    }
    if constexpr (PT) {
#pragma unroll
      for (int c0 = 0; c0 < BN / 2; c0 += 32) {
        uint32_t r[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) r[i] = fa_pack2(s[2 * (c0 + i)], s[2 * (c0 + i) + 1], fp16);
        tmem_st_32x32(t_lane + st * BN + c0, r);
      }
      tmem_wait_st();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar(st ? 15 : 13));
    } else {
    // ---- P (bf16) into shared memory: K-major, 128-byte swizzle: 16-byte chunk c of row r sits at c ^ (r & 7)
#pragma unroll
    for (int c = 0; c < BN / 64; ++c) {
#pragma unroll
      for (int q = 0; q < 8; ++q) {
        const int i0 = c * 64 + q * 8;
        uint4 v;
        v.x = fa_pack2(s[i0], s[i0 + 1], fp16); v.y = fa_pack2(s[i0 + 2], s[i0 + 3], fp16);
        v.z = fa_pack2(s[i0 + 4], s[i0 + 5], fp16); v.w = fa_pack2(s[i0 + 6], s[i0 + 7], fp16);
        const uint32_t addr = p_s + c * Q_SUB + row_l * 128 + ((q ^ (row_l & 7)) << 4);
        asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(addr), "r"(v.x), "r"(v.y), "r"(v.z), "r"(v.w) : "memory");
      }
    }
    fence_proxy_async_smem();   // generic-proxy writes -> visible to the tensor core's async proxy
    tc_fence_before();
    __syncwarp();
    if (lane == 0) mbar_arrive(bar(13));
    }
  }
  // ---- epilogue: O / l -> global, log-sum-exp
  if (ok && blocks.n > 0) {
    // not pv_done: a warp that has rescaled nothing lately may be two of its phases behind, which have the same parity
    ok = mbar_wait_warp(bar(0), 1, abort_flag, p.err, ERR_WAIT_TMEM_FULL);
    tc_fence_after();
  }
  float inv = l_sum > 0.f ? 1.f / l_sum : 0.f;
  const long long gate_row = (static_cast<long long>(b) * p.Sq + row) * p.ldg;
  const bool wide = p.gate != nullptr && p.gate_wide;
  if ((p.sink != nullptr || p.gate != nullptr) && row < p.Sq && l_sum > 0.f) {
    const long long gi = gate_row + h;
    inv = l_sum;
    if (p.sink != nullptr) {
      const float snk = fp16 ? __half2float(static_cast<const __half*>(p.sink)[h])
                             : __bfloat162float(static_cast<const __nv_bfloat16*>(p.sink)[h]);
      // m_ref is the running reference in log2 units; an overflowing sink term gives 1 / inf = 0
      inv += exp2f(snk * 1.4426950408889634f - m_ref);
    }
    if (p.gate != nullptr && !wide) {
      const float gate = fp16 ? __half2float(static_cast<const __half*>(p.gate)[gi])
                              : __bfloat162float(static_cast<const __nv_bfloat16*>(p.gate)[gi]);
      inv *= 1.f + exp2f(-gate * 1.4426950408889634f);
    }
    inv = 1.f / inv;
  }
  uint16_t* orow = reinterpret_cast<uint16_t*>(p.out) + b * p.o_sb + h * p.o_sh + static_cast<long long>(row) * p.o_ss;
#pragma unroll 1
  for (int c0 = 0; c0 < D; c0 += 32) {
    uint32_t r[32];
    if (blocks.n > 0 && ok) {
      tmem_ld_32x32(t_lane + O_COL + c0, r);
      tmem_wait_ld();
    } else {
#pragma unroll
      for (int i = 0; i < 32; ++i) r[i] = 0u;
    }
    if (row < p.Sq) {
#pragma unroll
      for (int i = 0; i < 32; i += 8) {
        if (c0 + i >= p.d_out) break;
        if (wide) {
          const uint4 g4 = *reinterpret_cast<const uint4*>(static_cast<const uint16_t*>(p.gate) + gate_row + h * p.d_out + c0 + i);
          const uint32_t gw[4] = {g4.x, g4.y, g4.z, g4.w};
#pragma unroll
          for (int u = 0; u < 4; ++u) {
            const float2 g = fp16 ? __half22float2(*reinterpret_cast<const __half2*>(&gw[u]))
                                  : __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gw[u]));
            r[i + 2 * u] = __float_as_uint(__fdividef(__uint_as_float(r[i + 2 * u]), 1.f + exp2f(-g.x * 1.4426950408889634f)));
            r[i + 2 * u + 1] = __float_as_uint(__fdividef(__uint_as_float(r[i + 2 * u + 1]), 1.f + exp2f(-g.y * 1.4426950408889634f)));
          }
        }
        uint4 v;
        v.x = fa_pack2(__uint_as_float(r[i]) * inv, __uint_as_float(r[i + 1]) * inv, fp16);
        v.y = fa_pack2(__uint_as_float(r[i + 2]) * inv, __uint_as_float(r[i + 3]) * inv, fp16);
        v.z = fa_pack2(__uint_as_float(r[i + 4]) * inv, __uint_as_float(r[i + 5]) * inv, fp16);
        v.w = fa_pack2(__uint_as_float(r[i + 6]) * inv, __uint_as_float(r[i + 7]) * inv, fp16);
        *reinterpret_cast<uint4*>(orow + c0 + i) = v;
      }
    }
  }
  if (row < p.Sq && p.lse) {
    const float lse = l_sum > 0.f ? (m_ref + log2f(l_sum)) * FA_LN2 : 0.f;
    p.lse[(static_cast<long long>(b) * p.H + h) * p.Sq + row] = lse;
  }
}

// PT = true: P goes back into TMEM (over the S buffer it came from, two bf16 per 32-bit column) and is the
// A operand of P V straight from tensor memory; PT = false: P goes through a swizzled shared-memory tile.
// CAP = true: capped scores, tanh(u) = 1 - 2 / (exp(2u) + 1) in 32-bit (absolute error about 2^-23 of the cap).
// Head sizes below D: the tensor maps are as wide as the heads, TMA fills the rest of a tile with zeros.
// DQ: columns of the query and key tiles, D: of the value tiles and the result. PARTS = true: the last sub-tiles of
// queries and keys have tensor maps of their own.
template <int DQ, int D, int BN, bool PT, bool CAP, bool PARTS>
__global__ void __launch_bounds__(FA_THREADS, 1)
fa_fwd_kernel(const __grid_constant__ CUtensorMap tq, const __grid_constant__ CUtensorMap tk,
              const __grid_constant__ CUtensorMap tv, const __grid_constant__ CUtensorMap tq2,
              const __grid_constant__ CUtensorMap tk2, const FaParams p) {
  constexpr int DC = DQ / 64, VC = D / 64;       // 64-column sub-tiles per row operand
  constexpr uint32_t Q_SUB = FA_BM * 128;        // bytes of one [128 x 64] sub-tile (Q and P)
  constexpr uint32_t KV_SUB = BN * 128;          // bytes of one [BN x 64] sub-tile (K and V)
  constexpr uint32_t Q_BYTES = DC * Q_SUB;
  constexpr uint32_t K_BYTES = DC * KV_SUB, V_BYTES = VC * KV_SUB;
  constexpr uint32_t P_BYTES = PT ? 0u : (BN / 64) * Q_SUB;
  constexpr uint32_t TMEM_COLS = 512;
  constexpr uint32_t O_COL = 2 * BN;             // S buffers at columns [0, BN) and [BN, 2 BN)
  static_assert(O_COL + D <= TMEM_COLS, "TMEM budget");

  extern __shared__ uint8_t fa_smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(fa_smem_raw) + 1023) & ~uintptr_t(1023));
  const uint32_t q_s = smem_u32(smem);
  const uint32_t k_s = q_s + Q_BYTES;            // 2 stages
  const uint32_t v_s = k_s + 2 * K_BYTES;        // 2 stages
  const uint32_t p_s = v_s + 2 * V_BYTES;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + Q_BYTES + 2 * (K_BYTES + V_BYTES) + P_BYTES);
  const uint32_t bar0 = smem_u32(bars);
  // 0 q_full, then the last P V | 1,2 k_full | 3,4 k_empty | 5,6 v_full | 7,8 v_empty | 9,10 s_full | 11,12 s_empty | 13 p_ready[0] |
  // 14 pv_done | 15 p_ready[1] (PT only: one per S/P buffer)
  auto bar = [&](int i) { return bar0 + 8u * i; };
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 16);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = blockIdx.z, h = blockIdx.y;
  const int q0 = (static_cast<int>(gridDim.x) - 1 - static_cast<int>(blockIdx.x)) * FA_BM;  // long (late) rows first
  const FaBlocks blocks(p, b, q0, BN);
  const int nblk = blocks.n;

  if (threadIdx.x == 0) {
    for (int i = 0; i < 16; ++i) {
      const bool four = (i == 11 || i == 12 || i == 13 || i == 15);  // arrivals from the 4 softmax warps
      mbar_init(bar(i), four ? 4 : 1);
    }
    *abort_flag = 0;
    fence_barrier_init();
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_slot), TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer
    if (lane == 0 && nblk > 0) {
      tma_prefetch_desc(&tq); tma_prefetch_desc(&tk); tma_prefetch_desc(&tv);
      mbar_expect_tx(bar(0), Q_BYTES);
#pragma unroll
      for (int c = 0; c < DC; ++c) {
        if (PARTS && c >= p.sub_first) tma_load_rows(q_s + c * Q_SUB, &tq2, bar(0), (c - p.sub_first) * 64, q0, h, b, p.q2_pos);
        else tma_load_rows(q_s + c * Q_SUB, &tq, bar(0), c * 64, q0, h, b, p.q_pos);
      }
      bool ok = true;
      const int hk = h / p.group;
      for (int j = 0; j < nblk && ok; ++j) {
        const int st = j & 1;
        const uint32_t ph = (j >> 1) & 1;
        const int n0 = blocks.start(j);
        ok = mbar_wait(bar(3 + st), ph ^ 1, abort_flag, p.err, ERR_WAIT_EMPTY);
        if (!ok) break;
        mbar_expect_tx(bar(1 + st), K_BYTES);
#pragma unroll
        for (int c = 0; c < DC; ++c) {
          const uint32_t dst = k_s + st * K_BYTES + c * KV_SUB;
          if (PARTS && c >= p.sub_first) tma_load_rows(dst, &tk2, bar(1 + st), (c - p.sub_first) * 64, n0, 0, b, p.k2_pos);
          else tma_load_rows(dst, &tk, bar(1 + st), c * 64, n0, hk, b, p.k_pos);
        }
        ok = mbar_wait(bar(7 + st), ph ^ 1, abort_flag, p.err, ERR_WAIT_EMPTY);
        if (!ok) break;
        mbar_expect_tx(bar(5 + st), V_BYTES);
#pragma unroll
        for (int c = 0; c < VC; ++c) tma_load_rows(v_s + st * V_BYTES + c * KV_SUB, &tv, bar(5 + st), c * 64, n0, hk, b, p.v_pos);
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    if (lane == 0 && nblk > 0) {
      const int fmt = p.fp16 ? 0 : 1;
      const uint32_t idesc_qk = make_idesc_f16(FA_BM, BN, fmt, 0, 0);
      const uint32_t idesc_pv = make_idesc_f16(FA_BM, D, fmt, 0, 1);
      bool ok = mbar_wait(bar(0), 0, abort_flag, p.err, ERR_WAIT_FULL);
      auto issue_qk = [&](int j) -> bool {
        const int st = j & 1;
        const uint32_t ph = (j >> 1) & 1;
        if (!mbar_wait(bar(1 + st), ph, abort_flag, p.err, ERR_WAIT_FULL)) return false;
        if (!mbar_wait(bar(11 + st), ph ^ 1, abort_flag, p.err, ERR_WAIT_TMEM_EMPTY)) return false;
        tc_fence_after();
#pragma unroll
        for (int kk = 0; kk < DQ / 16; ++kk) {
          const uint64_t da = make_smem_desc(q_s + (kk >> 2) * Q_SUB + (kk & 3) * 32, 16, 1024);
          const uint64_t db = make_smem_desc(k_s + st * K_BYTES + (kk >> 2) * KV_SUB + (kk & 3) * 32, 16, 1024);
          umma_f16(tmem_base + st * BN, da, db, idesc_qk, kk != 0);
        }
        umma_commit(bar(3 + st));   // K stage may be refilled once these MMAs have read it
        umma_commit(bar(9 + st));   // S_j is ready for the softmax warps
        return true;
      };
      if (ok) ok = issue_qk(0);
      for (int j = 0; j < nblk && ok; ++j) {
        if (j + 1 < nblk) {
          ok = issue_qk(j + 1);
          if (!ok) break;
        }
        const int st = j & 1;
        ok = mbar_wait(bar(5 + st), (j >> 1) & 1, abort_flag, p.err, ERR_WAIT_FULL);
        if (!ok) break;
        if (PT) ok = mbar_wait(bar(st ? 15 : 13), (j >> 1) & 1, abort_flag, p.err, ERR_WAIT_FULL);
        else ok = mbar_wait(bar(13), j & 1, abort_flag, p.err, ERR_WAIT_FULL);
        if (!ok) break;
        tc_fence_after();
#pragma unroll
        for (int ks = 0; ks < BN / 16; ++ks) {
          const uint64_t db = make_smem_desc(v_s + st * V_BYTES + ks * 2048, KV_SUB, 1024);
          if (PT) {
            umma_f16_ts(tmem_base + O_COL, tmem_base + st * BN + ks * 8, db, idesc_pv, (j | ks) != 0);
          } else {
            const uint64_t da = make_smem_desc(p_s + (ks >> 2) * Q_SUB + (ks & 3) * 32, 16, 1024);
            umma_f16(tmem_base + O_COL, da, db, idesc_pv, (j | ks) != 0);
          }
        }
        umma_commit(bar(7 + st));   // V stage free
        umma_commit(bar(14));       // O updated, P buffer reusable
        if (j + 1 == nblk) umma_commit(bar(0));
      }
    }
  } else {
    // ------------------------------------------------------------------ softmax / correction / epilogue
    fa_softmax_warps<BN, PT, CAP>(p, D, blocks, tmem_base, bar0, p_s, abort_flag, warp, lane, b, h, q0);
  }

  if (*abort_flag) {
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) {
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, TMEM_COLS);
  }
}

// ---------------------------------------------------------------------- wide keys
// Queries and keys of any width (`chunks` sub-tiles of 64 columns), one key head for all query heads, value heads per group: attention whose
// heads are mixed before the softmax, with the mix folded into the queries (grouped_attention.cu). All operands are sub-tiles of
// 128 rows x 64 columns, two of them to a 32 KB slot (a slot's hand-over costs the issuing thread about as much as four
// products take): the first FW_RESIDENT slots hold queries for good, everything else - keys, values, the rest of the queries -
// passes through a ring in the order in which the MMA warp uses it, Q K^T of block j + 1 ahead of P V of block j.
constexpr int FW_SLOTS = 7, FW_RESIDENT = 4;
constexpr uint32_t FW_SUB = 128 * 128, FW_SLOT = 2 * FW_SUB;

__global__ void __launch_bounds__(FA_THREADS, 1)
fa_wide_kernel(const __grid_constant__ CUtensorMap tq, const __grid_constant__ CUtensorMap tk, const __grid_constant__ CUtensorMap tv,
               const FaParams p, const int dim) {
  constexpr int BN = 128;
  constexpr uint32_t TMEM_COLS = 512, O_COL = 2 * BN;
  extern __shared__ uint8_t fa_smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(fa_smem_raw) + 1023) & ~uintptr_t(1023));
  const int chunks = (dim + 63) / 64, pairs = (chunks + 1) / 2, resident = min(pairs, FW_RESIDENT), ring = FW_SLOTS - resident;
  const int vc = (p.d_out + 63) / 64;
  const uint32_t q_s = smem_u32(smem), ring_s = q_s + resident * FW_SLOT;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + FW_SLOTS * FW_SLOT);
  const uint32_t bar0 = smem_u32(bars);
  // 0 q_full | 9.. as in fa_softmax_warps | 16 + i slot i full | 16 + FW_SLOTS + i slot i empty
  auto bar = [&](int i) { return bar0 + 8u * i; };
  constexpr int BARS = 16 + 2 * FW_SLOTS;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + BARS);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = blockIdx.z, h = blockIdx.y;
  const int q0 = (static_cast<int>(gridDim.x) - 1 - static_cast<int>(blockIdx.x)) * FA_BM;  // long (late) rows first
  const FaBlocks blocks(p, b, q0, BN);
  const int nblk = blocks.n;

  if (threadIdx.x == 0) {
    for (int i = 0; i < BARS; ++i) {
      const bool four = (i == 11 || i == 12 || i == 13 || i == 15);  // arrivals from the 4 softmax warps
      mbar_init(bar(i), four ? 4 : 1);
    }
    *abort_flag = 0;
    fence_barrier_init();
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_slot), TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  // the slots in turn; `phase` is the parity of the ring's current round
  struct Cursor {
    int slot = 0;
    uint32_t phase = 0;
    __device__ __forceinline__ void next(int ring) {
      if (++slot == ring) { slot = 0; phase ^= 1; }
    }
  };

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer
    if (lane == 0 && nblk > 0) {
      tma_prefetch_desc(&tq); tma_prefetch_desc(&tk); tma_prefetch_desc(&tv);
      const int first = min(chunks, 2 * resident);
      mbar_expect_tx(bar(0), first * FW_SUB);
      for (int c = 0; c < first; ++c) tma_load_rows(q_s + c * FW_SUB, &tq, bar(0), c * 64, q0, h, b, p.q_pos);
      Cursor at;
      bool ok = true;
      // sub-tiles c and (below `end`) c + 1 into the next slot
      auto load = [&](const CUtensorMap* map, int c, int end, int row, int head, const int* pos) {
        ok = mbar_wait(bar(16 + FW_SLOTS + at.slot), at.phase ^ 1, abort_flag, p.err, ERR_WAIT_EMPTY);
        if (!ok) return;
        const uint32_t full = bar(16 + at.slot), dst = ring_s + at.slot * FW_SLOT;
        const bool two = c + 1 < end;
        mbar_expect_tx(full, two ? FW_SLOT : FW_SUB);
        tma_load_rows(dst, map, full, c * 64, row, head, b, pos);
        if (two) tma_load_rows(dst + FW_SUB, map, full, c * 64 + 64, row, head, b, pos);
        at.next(ring);
      };
      auto keys = [&](int j) {
        const int n0 = blocks.start(j);
        for (int g = 0; g < pairs && ok; ++g) {
          if (g >= resident) load(&tq, 2 * g, chunks, q0, h, p.q_pos);
          if (ok) load(&tk, 2 * g, chunks, n0, 0, p.k_pos);
        }
      };
      keys(0);
      for (int j = 0; j < nblk && ok; ++j) {
        if (j + 1 < nblk) keys(j + 1);
        for (int c = 0; c < vc && ok; c += 2) load(&tv, c, vc, blocks.start(j), h / p.group, p.v_pos);
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    // The whole warp runs the loops, so that addresses and descriptors are warp-uniform; one lane issues.
    if (nblk > 0) {
      const int fmt = p.fp16 ? 0 : 1;
      const uint32_t idesc_qk = make_idesc_f16(FA_BM, BN, fmt, 0, 0);
      const uint32_t idesc_pv = make_idesc_f16(FA_BM, 128, fmt, 0, 1), idesc_pv1 = make_idesc_f16(FA_BM, 64, fmt, 0, 1);
      const uint64_t desc_k = make_smem_desc(0, 16, 1024), desc_v = make_smem_desc(0, FW_SUB, 1024);   // plus (address >> 4)
      const uint32_t q_at = q_s >> 4, ring_at = ring_s >> 4;
      constexpr uint32_t SLOT_AT = FW_SLOT >> 4, SUB_AT = FW_SUB >> 4;
      const bool issuer = elect_one();
      Cursor at;
      bool ok = mbar_wait(bar(0), 0, abort_flag, p.err, ERR_WAIT_FULL);
      auto issue_qk = [&](int j) -> bool {
        const int st = j & 1;
        if (!mbar_wait(bar(11 + st), ((j >> 1) & 1) ^ 1, abort_flag, p.err, ERR_WAIT_TMEM_EMPTY)) return false;
        tc_fence_after();
        const uint32_t dst = tmem_base + st * BN;
        for (int g = 0; g < pairs; ++g) {
          uint32_t a = q_at + g * SLOT_AT;
          int a_slot = -1;
          if (g >= resident) {
            if (!mbar_wait(bar(16 + at.slot), at.phase, abort_flag, p.err, ERR_WAIT_FULL)) return false;
            a_slot = at.slot;
            a = ring_at + at.slot * SLOT_AT;
            at.next(ring);
          }
          if (!mbar_wait(bar(16 + at.slot), at.phase, abort_flag, p.err, ERR_WAIT_FULL)) return false;
          const uint64_t da = desc_k + a, db = desc_k + (ring_at + at.slot * SLOT_AT);
          const int left = dim - g * 128;              // columns from this slot on
          if (issuer) {
            if (left >= 128) {
#pragma unroll
              for (int kk = 0; kk < 8; ++kk) {
                const uint32_t off = (kk >> 2) * SUB_AT + (kk & 3) * 2;
                umma_f16(dst, da + off, db + off, idesc_qk, (g | kk) != 0);
              }
            } else {
              for (int kk = 0; kk * 16 < left; ++kk) {
                const uint32_t off = (kk >> 2) * SUB_AT + (kk & 3) * 2;
                umma_f16(dst, da + off, db + off, idesc_qk, (g | kk) != 0);
              }
            }
            if (a_slot >= 0) umma_commit(bar(16 + FW_SLOTS + a_slot));   // the slots may be refilled once these MMAs have read them
            umma_commit(bar(16 + FW_SLOTS + at.slot));
            if (g + 1 == pairs) umma_commit(bar(9 + st));                // S_j is ready for the softmax warps
          }
          __syncwarp();
          at.next(ring);
        }
        return true;
      };
      if (ok) ok = issue_qk(0);
      for (int j = 0; j < nblk && ok; ++j) {
        if (j + 1 < nblk) {
          ok = issue_qk(j + 1);
          if (!ok) break;
        }
        const int st = j & 1;
        ok = mbar_wait(bar(st ? 15 : 13), (j >> 1) & 1, abort_flag, p.err, ERR_WAIT_FULL);
        if (!ok) break;
        tc_fence_after();
        for (int c = 0; c < vc && ok; c += 2) {
          ok = mbar_wait(bar(16 + at.slot), at.phase, abort_flag, p.err, ERR_WAIT_FULL);
          if (!ok) break;
          const uint64_t db = desc_v + (ring_at + at.slot * SLOT_AT);
          const uint32_t dst = tmem_base + O_COL + c * 64, src = tmem_base + st * BN;
          const uint32_t idesc = c + 1 < vc ? idesc_pv : idesc_pv1;
          if (issuer) {
#pragma unroll
            for (int ks = 0; ks < BN / 16; ++ks) umma_f16_ts(dst, src + ks * 8, db + ks * 128, idesc, (j | ks) != 0);
            umma_commit(bar(16 + FW_SLOTS + at.slot));
            if (c + 2 >= vc) umma_commit(bar(14));                       // O updated, P buffer reusable
            if (c + 2 >= vc && j + 1 == nblk) umma_commit(bar(0));
          }
          __syncwarp();
          at.next(ring);
        }
      }
    }
  } else {
    fa_softmax_warps<BN, true, false>(p, vc * 64, blocks, tmem_base, bar0, 0u, abort_flag, warp, lane, b, h, q0);
  }

  if (*abort_flag) {
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) {
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, TMEM_COLS);
  }
}

// ---------------------------------------------------------------------- host side
struct FaMaps {
  CUtensorMap q, k, v, q2, k2;                   // q2, k2: copies of q, k where there is no second part
};
template <int DQ, int D, int BN, bool PT, bool CAP, bool PARTS>
static int fa_launch_parts(const FaMaps& t, const FaParams& p, cudaStream_t stream) {
  constexpr size_t smem = FA_BM * DQ * 2 + 2 * BN * (DQ + D) * 2 + (PT ? 0 : FA_BM * BN * 2) + 16 * 8 + 16 + 1024;
  static_assert(smem <= 232448, "shared memory budget of one CTA");
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(fa_fwd_kernel<DQ, D, BN, PT, CAP, PARTS>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
    configured = true;
  }
  dim3 grid((p.Sq + FA_BM - 1) / FA_BM, p.H, p.B);
  fa_fwd_kernel<DQ, D, BN, PT, CAP, PARTS><<<grid, FA_THREADS, smem, stream>>>(t.q, t.k, t.v, t.q2, t.k2, p);
  return static_cast<int>(cudaGetLastError());
}
template <int D, int BN, bool PT, bool CAP = false>
static int fa_launch(const FaMaps& t, const FaParams& p, cudaStream_t stream) {
  return fa_launch_parts<D, D, BN, PT, CAP, false>(t, p, stream);
}

}  // namespace oslo

namespace oslo {
// what only some models have: a window's kept first keys, and a second part of queries and keys, q2 [B, H, Sq, rot] and
// k2 [B, Sk, rot] (one for all heads)
struct FaExtras {
  int keep_first = 0;
  const int* lead = nullptr;
  int gate_wide = 0;
  const void *q2 = nullptr, *k2 = nullptr;
  int rot = 0;
  long long q2_sb = 0, q2_sh = 0, q2_ss = 0, k2_sb = 0, k2_ss = 0;
};

static int flash_fwd_entry(const void* q, const void* k, const void* v, void* o, float* lse, const uint8_t* kpm,
                           const void* sink, const void* gate, long long ldg, int B, int H, int G, int Sq, int Sk, int dim, int vdim,
                           long long q_sb, long long q_sh, long long q_ss, long long k_sb, long long k_sh, long long k_ss,
                           long long v_sb, long long v_sh, long long v_ss, long long o_sb, long long o_sh, long long o_ss,
                           float scale, float softcap, int causal, int window, int dtype, int* err_word, cudaStream_t stream,
                           const FaExtras& x = FaExtras()) {
  if (B <= 0 || H <= 0 || Sq <= 0 || Sk <= 0 || G <= 0 || H % G) return -1;
  const bool parts = x.rot > 0;
  const int sub_first = (dim + 63) / 64, sub_all = sub_first + (x.rot + 63) / 64;
  const int widest = std::max(parts ? sub_all * 64 : dim, vdim);
  const int D = widest <= 64 ? 64 : (widest <= 128 ? 128 : 256);
  if (dim <= 0 || vdim <= 0 || widest > 256 || dim % 8 || vdim % 8) return -2;
  if (dtype != OSLO_DT_BF16 && dtype != OSLO_DT_FP16) return -3;
  if ((reinterpret_cast<uintptr_t>(o) & 15) || (o_sb % 8) || (o_sh % 8) || (o_ss % 8)) return -4;
  static thread_local bool ctx_bound = false;
  if (!ctx_bound) { cudaFree(nullptr); ctx_bound = true; }
  const bool fp16 = dtype == OSLO_DT_FP16;
  const bool narrow = parts && sub_all == 3 && vdim <= 128;    // 192 query and key columns, 128 value columns
  const int bn = D == 256 && !narrow ? 64 : 128;
  if (parts && (x.rot % 8 || softcap > 0.f)) return -2;
  if (x.gate_wide && (ldg % 8 || (reinterpret_cast<uintptr_t>(gate) & 15))) return -4;
  FaParams p;
  p.out = o; p.lse = lse; p.kpm = kpm;
  p.sink = sink; p.gate = gate; p.ldg = ldg; p.d_out = vdim; p.gate_wide = x.gate_wide;
  p.keep_first = window > 0 ? x.keep_first : 0; p.lead = x.lead; p.sub_first = sub_first;
  p.group = H / G; p.softcap = softcap;
  p.B = B; p.H = H; p.Sq = Sq; p.Sk = Sk;
  p.o_sb = o_sb; p.o_sh = o_sh; p.o_ss = o_ss;
  p.scale = scale; p.causal = causal; p.window = window; p.fp16 = fp16 ? 1 : 0; p.err = err_word;
  FaMaps t;
  int rc = make_qkv_map(&t.q, q, B, H, Sq, dim, q_sb, q_sh, q_ss, FA_BM, fp16, p.q_pos);
  if (rc) return rc;
  rc = make_qkv_map(&t.k, k, B, G, Sk, dim, k_sb, k_sh, k_ss, bn, fp16, p.k_pos);
  if (rc) return rc - 1000;
  rc = make_qkv_map(&t.v, v, B, G, Sk, vdim, v_sb, v_sh, v_ss, bn, fp16, p.v_pos);
  if (rc) return rc - 2000;
  t.q2 = t.q;
  t.k2 = t.k;
  if (parts) {
    rc = make_qkv_map(&t.q2, x.q2, B, H, Sq, x.rot, x.q2_sb, x.q2_sh, x.q2_ss, FA_BM, fp16, p.q2_pos);
    if (rc) return rc - 3000;
    // one head, so its stride only has to be valid
    rc = make_qkv_map(&t.k2, x.k2, B, 1, Sk, x.rot, x.k2_sb, x.k2_ss, x.k2_ss, bn, fp16, p.k2_pos);
    if (rc) return rc - 4000;
    if (D == 128) return fa_launch_parts<128, 128, 128, true, false, true>(t, p, stream);
    if (narrow) return fa_launch_parts<192, 128, 128, true, false, true>(t, p, stream);
    return fa_launch_parts<256, 256, 64, true, false, true>(t, p, stream);
  }
  if (softcap > 0.f) {
    if (D == 64) return fa_launch<64, 128, true, true>(t, p, stream);
    if (D == 128) return fa_launch<128, 128, true, true>(t, p, stream);
    return fa_launch<256, 64, true, true>(t, p, stream);
  }
  static const bool p_smem = [] { const char* e = getenv("OSLO_B200_ATTN_P_SMEM"); return e && e[0] == '1'; }();
  if (p_smem) {
    if (D == 64) return fa_launch<64, 128, false>(t, p, stream);
    if (D == 128) return fa_launch<128, 128, false>(t, p, stream);
    return fa_launch<256, 64, false>(t, p, stream);
  }
  if (D == 64) return fa_launch<64, 128, true>(t, p, stream);
  if (D == 128) return fa_launch<128, 128, true>(t, p, stream);
  return fa_launch<256, 64, true>(t, p, stream);
}
}  // namespace oslo

extern "C" int oslo_flash_fwd_sm100(const void* q, const void* k, const void* v, void* o, float* lse,
                                    const uint8_t* kpm, int B, int H, int Sq, int Sk, int D, long long q_sb,
                                    long long q_sh, long long q_ss, long long k_sb, long long k_sh, long long k_ss,
                                    long long v_sb, long long v_sh, long long v_ss, long long o_sb, long long o_sh,
                                    long long o_ss, float scale, int causal, int window, int dtype, int* err_word,
                                    cudaStream_t stream) {
  if (D != 64 && D != 128 && D != 256) return -2;
  return oslo::flash_fwd_entry(q, k, v, o, lse, kpm, nullptr, nullptr, 0, B, H, H, Sq, Sk, D, D, q_sb, q_sh, q_ss, k_sb, k_sh,
                               k_ss, v_sb, v_sh, v_ss, o_sb, o_sh, o_ss, scale, 0.f, causal, window, dtype, err_word, stream);
}

extern "C" int oslo_flash_sink_fwd_sm100(const void* q, const void* k, const void* v, void* o, const uint8_t* kpm,
                                         const void* sink, const void* gate, long long ldg, int B, int H, int G, int Sq, int Sk,
                                         int dim, int vdim, long long q_sb, long long q_sh, long long q_ss, long long k_sb,
                                         long long k_sh, long long k_ss, long long v_sb, long long v_sh, long long v_ss,
                                         long long o_sb, long long o_sh, long long o_ss, float scale, float softcap, int window,
                                         int keep_first, const int* lead, int gate_wide, const void* q2, long long q2_sb,
                                         long long q2_sh, long long q2_ss, const void* k2, long long k2_sb, long long k2_ss, int rot,
                                         int dtype, int* err_word, cudaStream_t stream) {
  oslo::FaExtras x;
  x.keep_first = keep_first; x.lead = lead; x.gate_wide = gate_wide; x.q2 = q2; x.k2 = k2; x.rot = q2 ? rot : 0;
  x.q2_sb = q2_sb; x.q2_sh = q2_sh; x.q2_ss = q2_ss; x.k2_sb = k2_sb; x.k2_ss = k2_ss;
  return oslo::flash_fwd_entry(q, k, v, o, nullptr, kpm, sink, gate, ldg, B, H, G, Sq, Sk, dim, vdim, q_sb, q_sh, q_ss, k_sb, k_sh,
                               k_ss, v_sb, v_sh, v_ss, o_sb, o_sh, o_ss, scale, softcap, 1, window, dtype, err_word, stream, x);
}

// q [B, H, Sq, dim], k [B, Sk, dim] (one head for all), v [B, G, Sk, vdim]
extern "C" int oslo_flash_wide_fwd_sm100(const void* q, const void* k, const void* v, void* o, const uint8_t* kpm, const void* sink,
                                         const void* gate, long long ldg, int gate_wide, int B, int H, int G, int Sq, int Sk, int dim,
                                         int vdim, long long q_sb, long long q_sh, long long q_ss, long long k_sb, long long k_ss,
                                         long long v_sb, long long v_sh, long long v_ss, long long o_sb, long long o_sh,
                                         long long o_ss, float scale, int window, int keep_first, const int* lead, int dtype,
                                         int* err_word, cudaStream_t stream) {
  using namespace oslo;
  if (B <= 0 || H <= 0 || Sq <= 0 || Sk < Sq || G <= 0 || H % G) return -1;
  if (dim <= 0 || vdim <= 0 || vdim > 256 || dim % 8 || vdim % 8) return -2;
  if (dtype != OSLO_DT_BF16 && dtype != OSLO_DT_FP16) return -3;
  if ((reinterpret_cast<uintptr_t>(o) & 15) || (o_sb % 8) || (o_sh % 8) || (o_ss % 8)) return -4;
  if (gate_wide && (ldg % 8 || (reinterpret_cast<uintptr_t>(gate) & 15))) return -4;
  static thread_local bool ctx_bound = false;
  if (!ctx_bound) { cudaFree(nullptr); ctx_bound = true; }
  const bool fp16 = dtype == OSLO_DT_FP16;
  FaParams p{};
  p.out = o; p.lse = nullptr; p.kpm = kpm; p.B = B; p.H = H; p.Sq = Sq; p.Sk = Sk;
  p.o_sb = o_sb; p.o_sh = o_sh; p.o_ss = o_ss;
  p.scale = scale; p.causal = 1; p.window = window; p.fp16 = fp16 ? 1 : 0; p.err = err_word; p.group = H / G; p.softcap = 0.f;
  p.sink = sink; p.gate = gate; p.ldg = ldg; p.d_out = vdim; p.gate_wide = gate_wide;
  p.keep_first = window > 0 ? keep_first : 0; p.lead = lead;
  FaMaps t;
  int rc = make_qkv_map(&t.q, q, B, H, Sq, dim, q_sb, q_sh, q_ss, FA_BM, fp16, p.q_pos);
  if (rc) return rc;
  rc = make_qkv_map(&t.k, k, B, 1, Sk, dim, k_sb, k_ss, k_ss, 128, fp16, p.k_pos);   // one head: its stride only has to be valid
  if (rc) return rc - 1000;
  rc = make_qkv_map(&t.v, v, B, G, Sk, vdim, v_sb, v_sh, v_ss, 128, fp16, p.v_pos);
  if (rc) return rc - 2000;
  constexpr size_t smem = FW_SLOTS * FW_SLOT + (16 + 2 * FW_SLOTS) * 8 + 16 + 1024;
  static_assert(smem <= 232448, "shared memory budget of one CTA");
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(fa_wide_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
    configured = true;
  }
  fa_wide_kernel<<<dim3((Sq + FA_BM - 1) / FA_BM, H, B), FA_THREADS, smem, stream>>>(t.q, t.k, t.v, p, dim);
  return static_cast<int>(cudaGetLastError());
}
