"""Shape / dtype ("fake tensor") implementations of the ``torch.ops.oslo_b200`` operators.

The reference's binding module only checks shapes and dtypes at call time
(oslo/fused_kernels/bindings/pybind_kernels.cpp:26-177). The kernels here are registered for the CUDA dispatch key,
so registering fake implementations lets the operators be traced under ``FakeTensorMode`` / ``torch.export`` /
``torch.compile`` graph capture without touching a GPU: each function returns empty tensors with the shapes,
dtypes and strides the kernels produce.
"""
from __future__ import annotations

import torch

_DONE = False
_FLAG_OUT_FP32 = 32


def register() -> None:
    """Idempotent; called once after the extension has been loaded."""
    global _DONE
    if _DONE:
        return
    _DONE = True
    reg = torch.library.register_fake

    @reg("oslo_b200::gemm")
    def _(a, b, a_mn, b_mn, bias, aux, out, aux_out, flags, alpha):
        if out is not None:
            return out
        m = a.size(1) if a_mn else a.size(0)
        n = b.size(1) if b_mn else b.size(0)
        return a.new_empty((m, n), dtype=torch.float32 if (flags & _FLAG_OUT_FP32) else a.dtype)

    @reg("oslo_b200::gemm_small_m")
    def _(a, b, b_mn, bias, gelu_from):
        return a.new_empty((a.size(0), b.size(1) if b_mn else b.size(0)))

    @reg("oslo_b200::gemv_rows")
    def _(x1, x2, w, bias, gelu_from, res=None):
        return x1.new_empty((x1.size(0), w.size(0)))

    @reg("oslo_b200::layernorm_fwd")
    def _(x, w, b, eps):
        rows = x.numel() // max(x.size(-1), 1)
        stat = x.new_empty((rows,), dtype=torch.float32)
        return torch.empty_like(x), stat, torch.empty_like(stat)

    @reg("oslo_b200::layernorm_bwd")
    def _(dy, x, w, mean, rstd):
        return torch.empty_like(x), torch.empty_like(w), torch.empty_like(w)

    @reg("oslo_b200::bias_gelu_fwd")
    def _(x, bias):
        return torch.empty_like(x)

    @reg("oslo_b200::bias_gelu_bwd")
    def _(dy, x, bias):
        return torch.empty_like(x)

    @reg("oslo_b200::colsum")
    def _(x):
        return x.new_empty((x.size(-1),), dtype=torch.float32)

    @reg("oslo_b200::rotary")
    def _(x, positions, rotary_dim, base, inverse):
        return torch.empty_like(x)

    @reg("oslo_b200::flash_fwd")
    def _(q, k, v, scale, causal, window, kpm, impl=1):
        b, h, sq, d = q.shape
        o = q.new_empty((b, sq, h, d)).permute(0, 2, 1, 3)     # [B, H, S, D] view of a [B, S, H, D] buffer
        return o, q.new_empty((b, h, sq), dtype=torch.float32)

    @reg("oslo_b200::flash_bwd")
    def _(dout, q, k, v, o, lse, scale, causal, window, kpm, impl=1):
        return (torch.empty_strided(q.shape, q.stride(), dtype=q.dtype, device=q.device),
                torch.empty_strided(k.shape, k.stride(), dtype=k.dtype, device=k.device),
                torch.empty_strided(v.shape, v.stride(), dtype=v.dtype, device=v.device))

    @reg("oslo_b200::decode_attn")
    def _(q, kc, vc, lengths, scale, window):
        return torch.empty_like(q)

    @reg("oslo_b200::causal_softmax_fwd")
    def _(x, scale):
        return torch.empty_like(x)

    @reg("oslo_b200::masked_softmax_fwd")
    def _(x, mask, scale):
        return torch.empty_like(x)

    @reg("oslo_b200::softmax_bwd")
    def _(y, dy, scale):
        return torch.empty_like(y)

    @reg("oslo_b200::ce_stats")
    def _(logits, labels, vocab_start):
        s = logits.new_empty((logits.size(0),), dtype=torch.float32)
        return s, torch.empty_like(s), torch.empty_like(s)

    @reg("oslo_b200::sumsq")
    def _(x):
        return x.new_empty((1,), dtype=torch.float32)

    @reg("oslo_b200::gemm_ce_stats")
    def _(a, b, b_mn, bias, labels, vocab_start):
        s = a.new_empty((a.size(0),), dtype=torch.float32)
        return s, torch.empty_like(s), torch.empty_like(s)

    @reg("oslo_b200::gemm_ce_grad")
    def _(a, b, b_mn, bias, labels, vocab_start, lse, scale):
        return a.new_empty((a.size(0), b.size(1) if b_mn else b.size(0)))

    @reg("oslo_b200::error_word")
    def _(like):
        return like.new_empty((1,), dtype=torch.int32)

    @reg("oslo_b200::bias_dropout_residual")
    def _(x, bias, residual, p, seed, mode):
        return torch.empty_like(x)

    @reg("oslo_b200::rotary_")
    def _(x, positions, heads, head_dim, rotary_dim, base, inverse):
        return x

    @reg("oslo_b200::ce_grad_")
    def _(logits, labels, vocab_start, lse, scale):
        return logits

    @reg("oslo_b200::adam_step")
    def _(p, g, m, v, p_lp, lr, beta1, beta2, eps, wd, step, grad_scale, inv_scale):
        return None

    @reg("oslo_b200::ngram_ban_")
    def _(tokens, lprobs, n):
        return lprobs

    @reg("oslo_b200::rotary_append")
    def _(q, k, v, kc, vc, lengths, write_index, rotary_dim, base):
        return q.new_empty((kc.size(0), kc.size(1), kc.size(3)))

    @reg("oslo_b200::wait_probe")
    def _(flag, target, limit_ms):
        return flag.new_empty((1,), dtype=torch.int64)

    # collectives over symmetric memory: the data moves between GPUs inside the kernels; for tracing only the local
    # outputs matter (in-place operators return nothing)
    @reg("oslo_b200::gemm_comm")
    def _(a, b, a_mn, b_mn, bias, aux, aux_out, out, flags, alpha, M, N, K, peer_bufs_dev, own_buf, mc_base, data_off,
          flag_off, flag_bytes, rank, world, epoch, done_base, mode, use_multimem, trace):
        return 0

    @reg("oslo_b200::vocab_embed")
    def _(ids, weight, lo, hi, peer_ptrs_dev, mc_ptr, signal_ptrs_dev, counters, half_bytes, rank, world, use_multimem):
        return weight.new_empty((ids.numel(), weight.size(1)))

    @reg("oslo_b200::allreduce_oneshot")
    def _(x, peer_ptrs_dev, mc_ptr, signal_ptrs_dev, counters, stage_off, half_bytes, rank, world, use_multimem):
        return None

    @reg("oslo_b200::allreduce_symm")
    def _(peer_ptrs_dev, mc_ptr, signal_ptrs_dev, out, numel, rank, world, use_multimem):
        return None

    @reg("oslo_b200::ce_combine")
    def _(mx, se, tg, peer_ptrs_dev, signal_ptrs_dev, counters, cap, rank, world):
        return None

    @reg("oslo_b200::dp_reduce_scatter")
    def _(like, peer_ptrs_dev, mc_ptr, signal_ptrs_dev, lo, hi, shard, rank, world, use_multimem):
        return None

    @reg("oslo_b200::dp_all_gather")
    def _(like, peer_ptrs_dev, mc_ptr, signal_ptrs_dev, lo, hi, shard, rank, world, use_multimem):
        return None


    @reg("oslo_b200::rms_norm")
    def _(x, w, eps, offset):
        return w.new_empty(x.shape)

    @reg("oslo_b200::residual_join")
    def _(x, y, slots, slot_weights, gate, gate_bias, w_post, w_next, eps):
        return torch.empty_like(x), y.new_empty((x.size(0) if w_next is not None else 0, x.size(1)))

    @reg("oslo_b200::silu_mul")
    def _(gate, up):
        return gate.new_empty(gate.shape)

    @reg("oslo_b200::recurrence")
    def _(q, f, v, f_bias, lower, keep, state, batch, heads, dim, vdim, chunks=0):
        return q.new_empty((batch, q.size(0) // batch, heads, vdim), dtype=torch.float32)

    @reg("oslo_b200::recurrence_step")
    def _(q, f, v, f_bias, lower, norm_w, keep, state, eps, heads, dim, vdim):
        return q.new_empty((q.size(0), heads * vdim))

    @reg("oslo_b200::sink_gate")
    def _(o, lse, sink, gate, vdim):
        return o.new_empty((o.size(0) * o.size(2), o.size(1) * vdim))

    @reg("oslo_b200::flash_sink_fwd")
    def _(q, k, v, kpm, sink, gate, scale, softcap, window=0, keep_first=0, lead=None, q2=None, k2=None):
        return q.new_empty((q.size(0) * q.size(2), q.size(1) * v.size(3)))

    @reg("oslo_b200::sink_attention")
    def _(q, k, v, keep, sink, gate, scale, softcap, window=0, keep_first=0, lead=None):
        return q.new_empty((q.size(0) * q.size(1), q.size(2) * v.size(3)))

    @reg("oslo_b200::latent_prep")
    def _(cq, wq, ckv, wkv, cache, lengths, eps, positions=None, freq=None, rows=False):
        return cq.new_empty(cq.shape), cq.new_empty((cq.size(0) if rows and ckv is not None else 0, 0 if wkv is None else wkv.numel()))

    @reg("oslo_b200::rotate_halves_")
    def _(q, positions, freq):
        return q

    @reg("oslo_b200::latent_decode")
    def _(q, w_uk, w_uv, cache, lengths, keep, sink, gate, scale, heads, positions=None, freq=None):
        return q.new_empty((q.size(0), w_uv.size(0)))

    @reg("oslo_b200::moe_route")
    def _(h, w, bias, logits, top, scored=0):
        return h.new_empty((h.size(0), top), dtype=torch.int32), h.new_empty((h.size(0), top), dtype=torch.float32)

    @reg("oslo_b200::moe_plan")
    def _(h, idx, experts, scale=None):
        tiles = (idx.numel() + 127) // 128 + min(experts, idx.numel())
        return (torch.empty_like(idx), h.new_empty((tiles * 128, h.size(1))), idx.new_empty((tiles,)), idx.new_empty((1,)))

    @reg("oslo_b200::moe_grouped")
    def _(rows, w, tile_group, n_tiles, unit, limit=0.0, alpha=1.0):
        return rows.new_empty((rows.size(0), w.size(1) // (2 if unit >= 2 else 1)))

    @reg("oslo_b200::moe_few")
    def _(x, idx, w, per_row, unit, limit=0.0, alpha=1.0, scale=None):
        return x.new_empty((idx.numel(), w.size(1) // (2 if unit >= 2 else 1)))

    @reg("oslo_b200::clamped_glu")
    def _(gate, up, limit, alpha):
        return gate.new_empty(gate.shape)

    @reg("oslo_b200::branch_join")
    def _(x, y, w, factor, normed, slots, top, mult, eps, w1, w2, copy=False, conv_w=None, prev=None, keep=None):
        rows, cols = x.shape
        outs = (w1 is not None or copy, w2 is not None, conv_w is not None)
        return (torch.empty_like(x), *(y[0].new_empty((rows if there else 0, cols)) for there in outs))

    @reg("oslo_b200::token_gate")
    def _(z, ids, table, first):
        return z.new_empty(z.shape)

    @reg("oslo_b200::gated_rms_norm")
    def _(o, w, gate, eps, group, act, z=None, m=None):
        return w.new_empty(o.shape)

    @reg("oslo_b200::hyper_join")
    def _(x, y, slots, weights, choice, experts, own, shared, gate, w_out, mix, w_in, w_norm, eps, scale):
        rows, n, cols = x.shape
        return x.new_empty((rows if y is not None else 0, n, cols)), w_norm.new_empty((rows, cols))

    @reg("oslo_b200::memory_gates")
    def _(z, bias, cap, keep, top, batch):
        heads, s = z.size(1) // 2, z.size(0) // batch
        return (*(z.new_empty((batch, heads, s)) for _ in range(3)), z.new_empty((z.size(0), heads)))

    @reg("oslo_b200::memory_recurrence")
    def _(q, k, v, read, write, start, q_scale, keep, state, batch, heads, dim, vdim, chunks=0):
        return q.new_empty((q.size(0), heads * vdim), dtype=torch.float32), q.new_empty((q.size(0), heads), dtype=torch.float32)

    @reg("oslo_b200::memory_step")
    def _(q, k, v, x, w, bias, cap, gate, norm_w, keep, state, top, q_scale, eps, heads, dim, vdim):
        return q.new_empty((q.size(0), heads * vdim))

    @reg("oslo_b200::gemv_stacked")
    def _(x, w):
        return x.new_empty((x.size(0), x.size(1), w.size(1)))

    @reg("oslo_b200::decayed_recurrence")
    def _(q, k, v, decay, keep, state, batch, heads, dim, vdim, chunks=0):
        return q.new_empty((batch, q.size(0) // batch, heads, vdim), dtype=torch.float32)

    @reg("oslo_b200::bonus_recurrence")
    def _(q, k, v, z, w0, u, keep, state, batch, heads, dim, vdim, chunks=0):
        return q.new_empty((batch, q.size(0) // batch, heads, vdim), dtype=torch.float32)

    @reg("oslo_b200::decayed_step")
    def _(q, k, v, decay, keep, state, heads, dim, vdim):
        return q.new_empty((q.size(0), heads * vdim), dtype=torch.float32)

    @reg("oslo_b200::bonus_step")
    def _(r, k, v, t, w2, w0, u, norm_w, gate, keep, state, eps, heads, dim, vdim):
        return r.new_empty((r.size(0), heads * vdim))

    @reg("oslo_b200::qkv_prep")
    def _(q, k, v, wq, wk, eps, positions, freq, kc, vc, lengths):
        return q.new_empty((kc.size(0), q.size(0) // kc.size(0), q.size(1) // kc.size(3), kc.size(3)))

    @reg("oslo_b200::head_prep")
    def _(q, k, v, wq, wk, eps, positions, freq, halves, amplitude, talk, kc, vc, lengths):
        b, g, _, d = kc.shape
        return q.new_empty((b, q.size(0) // b, q.size(1) // d, d if talk is None else g * d))

    @reg("oslo_b200::wide_decode_fits")
    def _(like, heads, value_heads, dim, vdim):
        return True

    @reg("oslo_b200::flash_wide_fwd")
    def _(q, k, v, kpm, sink, gate, scale, window=0, keep_first=0, lead=None):
        return q.new_empty((q.size(0) * q.size(2), q.size(1) * v.size(3)))

    @reg("oslo_b200::grouped_decode")
    def _(q, kc, vc, lengths, keep, sink, scale, softcap, gate=None, window=0, keep_first=0, lead=None, value_heads=1):
        return q.new_empty((q.size(0), q.size(1) * (vc.size(3) // value_heads)))

    @reg("oslo_b200::token_shift")
    def _(h, mu, batch, keep, prev):
        return h.new_empty((mu.size(0), h.size(0), h.size(1)))

    @reg("oslo_b200::causal_conv")
    def _(x, w, bias, batch, keep, prev, silu=False, residual=False):
        return x.new_empty(x.shape)

    @reg("oslo_b200::selective_scan")
    def _(x, dt, dt_bias, a_log, b, c, d, z, batch, keep, state, chunks=0):
        return x.new_empty(x.shape)

    @reg("oslo_b200::scan_step")
    def _(x, dt, w_dt, dt_bias, a_log, b, c, d, z, keep, state):
        return x.new_empty(x.shape)
