"""Public op functions: dispatch between the sm_100a kernels and the PyTorch statements."""
from __future__ import annotations

import math
from typing import Optional, Tuple

import torch
from torch import Tensor

from . import reference as ref

_GELU_NAMES = ("gelu", "gelu_new", "gelu_tanh", "gelu_pytorch_tanh")


def _k(x: Tensor) -> bool:
    from . import use_kernels
    return use_kernels(x)


def linear(x: Tensor, weight: Tensor, bias: Optional[Tensor] = None, reversed: bool = False,
           activation: Optional[str] = None) -> Tensor:
    """``act(x @ W.T + b)`` (or ``x @ W`` when ``reversed``). bf16/fp16 CUDA inputs use the tcgen05 GEMM."""
    if _k(x):
        from . import cuda_ops
        return cuda_ops.linear(x, weight, bias, reversed, activation)
    return ref.linear(x, weight, bias, reversed, activation)


def layer_norm(x: Tensor, weight: Tensor, bias: Optional[Tensor], eps: float = 1e-5) -> Tensor:
    if _k(x):
        from . import cuda_ops
        return cuda_ops.layer_norm(x, weight, bias, eps)
    return ref.layer_norm(x, weight, bias, eps)


def bias_gelu(x: Tensor, bias: Optional[Tensor] = None) -> Tensor:
    if _k(x):
        from . import cuda_ops
        return cuda_ops.bias_gelu(x, bias)
    return ref.bias_gelu(x, bias)


def bias_dropout_residual(x: Tensor, bias: Optional[Tensor] = None, residual: Optional[Tensor] = None,
                          p: float = 0.0, training: bool = False) -> Tensor:
    if _k(x):
        from . import cuda_ops
        return cuda_ops.bias_dropout_residual(x, bias, residual, p, training)
    return ref.bias_dropout_residual(x, bias, residual, p, training)


def rotary_interleaved(x: Tensor, positions: Tensor, rotary_dim: int, base: float = 10000.0) -> Tensor:
    """GPT-J rotary on ``[B, S, heads, D]`` with integer ``positions`` ``[B, S]``."""
    if _k(x):
        from . import cuda_ops
        return cuda_ops.rotary_interleaved(x, positions, rotary_dim, base)
    return ref.rotary_interleaved(x, positions, rotary_dim, base)


def attention(q: Tensor, k: Tensor, v: Tensor, causal: bool = True, window: Optional[int] = None,
              scale: Optional[float] = None, key_padding_mask: Optional[Tensor] = None,
              dropout_p: float = 0.0, training: bool = False) -> Tensor:
    """Flash-style attention on ``[B, heads, S, D]`` (any strides with contiguous ``D``)."""
    if scale is None:
        scale = 1.0 / math.sqrt(q.size(-1))
    if _k(q) and not (dropout_p > 0.0 and training):
        from . import cuda_ops
        if cuda_ops.flash_supported(q, k, v):
            return cuda_ops.flash_attention(q, k, v, causal, window, scale, key_padding_mask)
    return ref.attention(q, k, v, causal, window, scale, key_padding_mask, dropout_p, training)


def decode_attention(q: Tensor, k_cache: Tensor, v_cache: Tensor, lengths: Tensor, scale: float,
                     window: Optional[int] = None) -> Tensor:
    """One-query attention over a static KV cache.

    ``q``: ``[B, heads, D]``; caches ``[B, heads, T_max, D]``; ``lengths``: ``[B]`` valid keys per row
    (the query sits at position ``lengths - 1``).
    """
    if _k(q):
        from . import cuda_ops
        return cuda_ops.decode_attention(q, k_cache, v_cache, lengths, scale, window)
    B, H, T, D = k_cache.shape
    s = torch.einsum("bhd,bhtd->bht", q.float(), k_cache.float()) * scale
    pos = torch.arange(T, device=q.device)[None, :]
    keep = pos < lengths[:, None]
    if window is not None:
        keep &= pos > (lengths[:, None] - 1 - window)
    s = s.masked_fill(~keep[:, None, :], torch.finfo(torch.float32).min)
    p = torch.softmax(s, dim=-1)
    return torch.einsum("bht,bhtd->bhd", p, v_cache.float()).to(q.dtype)


def scaled_upper_triang_masked_softmax(x: Tensor, scale: float = 1.0) -> Tensor:
    if _k(x):
        from . import cuda_ops
        return cuda_ops.causal_softmax(x, scale)
    return _RefCausalSoftmax.apply(x, scale)


def scaled_masked_softmax(x: Tensor, mask: Tensor, scale: float = 1.0) -> Tensor:
    if _k(x):
        from . import cuda_ops
        return cuda_ops.masked_softmax(x, mask, scale)
    return ref.scaled_masked_softmax(x, mask, scale)


class _RefCausalSoftmax(torch.autograd.Function):
    @staticmethod
    def forward(ctx, x, scale):
        y = ref.scaled_upper_triang_masked_softmax(x, scale)
        ctx.save_for_backward(y)
        ctx.scale = scale
        return y

    @staticmethod
    def backward(ctx, dy):
        (y,) = ctx.saved_tensors
        return ref.softmax_backward(y, dy, ctx.scale), None


def cross_entropy(logits: Tensor, labels: Tensor, ignore_index: int = -100) -> Tensor:
    """Mean cross-entropy over rows of ``[N, V]`` logits with fp32 math."""
    if _k(logits):
        from . import cuda_ops
        return cuda_ops.cross_entropy(logits, labels, ignore_index)
    return ref.cross_entropy(logits, labels, ignore_index)


def linear_cross_entropy(hidden: Tensor, weight: Tensor, bias: Optional[Tensor], labels: Tensor,
                         ignore_index: int = -100, chunk_rows: int = 4096) -> Tensor:
    """LM-head projection fused with the loss, never holding more than ``chunk_rows`` rows of logits.

    ``hidden``: ``[N, H]``, ``weight``: ``[V, H]``, ``labels``: ``[N]`` (already shifted). Returns the
    mean loss over rows whose label is not ``ignore_index``.
    """
    if _k(hidden):
        from . import cuda_ops
        return cuda_ops.linear_cross_entropy(hidden, weight, bias, labels, ignore_index, chunk_rows)
    logits = ref.linear(hidden, weight, bias)
    return ref.cross_entropy(logits, labels, ignore_index)


def ban_repeated_ngrams(tokens: Tensor, lprobs: Tensor, n: int) -> Tensor:
    if _k(lprobs):
        from . import cuda_ops
        return cuda_ops.ban_repeated_ngrams(tokens, lprobs, n)
    return ref.ban_repeated_ngrams(tokens, lprobs, n)


# ---------------------------------------------------------------------------------------------------------------
# The kernels behind the functions below have no backward: with gradients on, the differentiable statement runs.
def _kn(x: Tensor, *others: Optional[Tensor]) -> bool:
    if torch.is_grad_enabled() and (x.requires_grad or any(t is not None and t.requires_grad for t in others)):
        return False
    return _k(x)


def rms_norm(x: Tensor, w: Tensor, eps: float, offset: float = 0.0) -> Tensor:
    """``x / sqrt(mean(x^2) + eps) * (offset + w)`` with fp32 math, in ``w``'s dtype; ``x`` is fp32 or has ``w``'s dtype."""
    if _kn(x, w):
        from . import cuda_ops
        return cuda_ops.rms_norm(x, w, eps, offset)
    return ref.rms_norm(x, w, eps, offset)


def residual_join(x: Tensor, y: Tensor, gate: Tensor, gate_bias: Tensor, w_post: Tensor, w_next: Optional[Tensor],
                  eps: float, slots: Optional[Tensor] = None,
                  slot_weights: Optional[Tensor] = None) -> Tuple[Tensor, Optional[Tensor]]:
    """Gate a sublayer's result, norm it, add it to the fp32 residual stream and norm the sum for the next sublayer: one
    pass over the rows. See ``reference.residual_join``."""
    if _kn(x, y, gate, gate_bias, w_post, w_next, slot_weights):
        from . import cuda_ops
        return cuda_ops.residual_join(x, y, gate, gate_bias, w_post, w_next, eps, slots, slot_weights)
    return ref.residual_join(x, y, gate, gate_bias, w_post, w_next, eps, slots, slot_weights)


def silu_mul(gate: Tensor, up: Tensor) -> Tensor:
    if _kn(gate, up):
        from . import cuda_ops
        return cuda_ops.silu_mul(gate, up)
    return ref.silu_mul(gate, up)


def gated_recurrence(q: Tensor, f: Tensor, v: Tensor, f_bias: Tensor, lower: Tensor, norm_w: Tensor, eps: float, batch: int,
                     heads: int, keep: Optional[Tensor] = None, state: Optional[Tensor] = None) -> Tensor:
    """``reference.recurrence`` followed by the RMS norm of every head's output; ``state`` (fp32, updated in place) carries the
    sequence on. ``[batch * S, heads * vdim]`` in ``norm_w``'s dtype."""
    if _kn(q, f, v, f_bias, lower, norm_w):
        from . import cuda_ops
        return cuda_ops.gated_recurrence(q, f, v, f_bias, lower, norm_w, eps, batch, heads, keep, state)
    dim, vdim = q.size(1) // heads, v.size(1) // heads
    o, final = ref.recurrence(q, f, v, f_bias, lower, keep, state, batch, heads, dim, vdim)
    if state is not None:
        state.copy_(final.detach())
    return ref.rms_norm(o, norm_w, eps).reshape(-1, heads * vdim)


def sink_attention(q: Tensor, k: Tensor, v: Tensor, keep: Optional[Tensor], sink: Optional[Tensor], gate: Optional[Tensor],
                   scale: float, softcap: float = 0.0, window: int = 0, keep_first: int = 0, lead: Optional[Tensor] = None,
                   q_rot: Optional[Tensor] = None, k_rot: Optional[Tensor] = None) -> Tensor:
    """``reference.sink_attention`` without the weights."""
    if _kn(q, k, v, sink, gate, q_rot, k_rot):
        from . import cuda_ops
        return cuda_ops.sink_attention(q, k, v, keep, sink, gate, scale, softcap, window, keep_first, lead, q_rot, k_rot)
    return ref.sink_attention(q, k, v, keep, sink, gate, scale, softcap, window, keep_first, lead, q_rot, k_rot)[0]


def latent_decode(q: Tensor, w_uk: Tensor, w_uv: Tensor, cache: Tensor, lengths: Tensor, keep: Optional[Tensor],
                  sink: Optional[Tensor], gate: Tensor, scale: float, heads: int, positions: Optional[Tensor] = None,
                  freq: Optional[Tensor] = None) -> Tensor:
    if _kn(q, w_uk, w_uv, cache, sink, gate):
        from . import cuda_ops
        return cuda_ops.latent_decode(q, w_uk, w_uv, cache, lengths, keep, sink, gate, scale, heads, positions, freq)
    return ref.latent_decode(q, w_uk, w_uv, cache, lengths, keep, sink, gate, scale, heads, positions, freq)


def moe_route(h: Tensor, w: Tensor, bias: Optional[Tensor], top: int, scored=False, fused: bool = True) -> Tuple[Tensor, Tensor]:
    if fused and _kn(h, w, bias):
        from . import cuda_ops
        return cuda_ops.moe_route(h, w, bias, top, scored)
    return ref.moe_route(h, w, bias, top, scored)


def moe_experts(h: Tensor, idx: Tensor, up: Tensor, down: Tensor, unit: str = "relu2", limit: float = 0.0, alpha: float = 1.702,
                scale: Optional[Tensor] = None, fused: bool = True) -> Tuple[Tensor, Optional[Tensor]]:
    """The chosen experts' results (``reference.moe_experts``), one row per (token, choice), and where those rows are (``None``: row
    ``token * top + choice``); the step that joins the residual stream adds them up. Rows of choices that are no expert hold anything."""
    if fused and _kn(h, up, down, scale):
        from . import cuda_ops
        return cuda_ops.moe_experts(h, idx, up, down, unit, limit, alpha, scale)
    return ref.moe_experts(h, idx, up, down, unit, limit, alpha, scale), None


def hyper_join(x: Tensor, result: Optional[ref.SublayerResult], w_out: Optional[Tensor], mix: Optional[Tensor],
               w_in: Optional[Tensor], w_norm: Tensor, eps: float, scale: float = 1.0, fused: bool = True) -> Tuple[Tensor, Tensor]:
    """Residual streams take a sublayer's result and the next sublayer's input is read from them: one pass over the rows. See
    ``reference.hyper_join``."""
    mine = () if result is None else (result.y, result.weights, result.h, result.shared, result.shared_gate)
    if fused and _kn(x, w_out, mix, w_in, w_norm, *mine):
        from . import cuda_ops
        return cuda_ops.hyper_join(x, result, w_out, mix, w_in, w_norm, eps, scale)
    return ref.hyper_join(x, result, w_out, mix, w_in, w_norm, eps, scale)


def linear_fp32(x: Tensor, weight: Tensor, fused: bool = True) -> Tensor:
    """``x @ W.T`` with a 32-bit result whatever the storage type: what enters a decay or a step size is not rounded to 16 bits."""
    if fused and _kn(x, weight):
        from . import cuda_ops
        return cuda_ops.linear_fp32(x, weight)
    return torch.matmul(x, weight.t()).to(torch.float32)


def stacked_linear(x: Tensor, weight: Tensor, fused: bool = True) -> Tuple[Tensor, ...]:
    """``x[i] @ W[i].T`` for every part ``i``: ``x`` ``[P, rows, in]``, ``weight`` ``[P, out, in]``."""
    if fused and _kn(x, weight):
        from . import cuda_ops
        return cuda_ops.stacked_linear(x, weight)
    return torch.matmul(x, weight.transpose(1, 2)).unbind(0)


def branch_join(x: Tensor, branches, mult: float, eps: float, w_next, copy: Optional[torch.dtype] = None, conv=None, fused: bool = True):
    """Add the results of parallel branches to the fp32 residual stream and norm the sum once per weight of ``w_next``, or copy it: one
    pass over the rows. See ``reference.branch_join``. ``conv`` ``(weight, state, keep)``, with one norm and rows that are single tokens:
    a second result, ``reference.causal_conv`` of the norm with ``residual`` (``state``, or ``None``, is updated)."""
    if fused and _kn(x, *(t for b in branches for t in b[:2]), *w_next):
        from . import cuda_ops
        return cuda_ops.branch_join(x, branches, mult, eps, w_next, copy, conv)
    x, out = ref.branch_join(x, branches, mult, eps, w_next, copy)
    if conv is not None:
        weight, state, keep = conv
        out.append(causal_conv(out[0], weight, None, x.size(0), keep, state, residual=True, fused=False))
    return x, out


def token_gate(z: Tensor, ids: Tensor, table: Tensor, first: int, fused: bool = True) -> Tensor:
    if fused and _kn(z, table):
        from . import cuda_ops
        return cuda_ops.token_gate(z, ids, table, first)
    return ref.token_gate(z, ids, table, first)


def clamped_glu(gate: Tensor, up: Tensor, limit: float, alpha: float, fused: bool = True) -> Tensor:
    if fused and _kn(gate, up):
        from . import cuda_ops
        return cuda_ops.clamped_glu(gate, up, limit, alpha)
    return ref.clamped_glu(gate, up, limit, alpha)


def gated_rms_norm(o: Tensor, w: Tensor, gate: Tensor, eps: float, group: int, act: str,
                   normalizer: Optional[Tuple[Tensor, Tensor]] = None, fused: bool = True) -> Tensor:
    if fused and _kn(o, w, gate):
        from . import cuda_ops
        return cuda_ops.gated_rms_norm(o, w, gate, eps, group, act, normalizer)
    return ref.gated_rms_norm(o, w, gate, eps, group, act, normalizer)


# ``state`` / ``prev`` of the functions below (fp32) carry a sequence on: read, and updated in place.
def decayed_attention(q: Tensor, k: Tensor, v: Tensor, decay: Tensor, keep: Optional[Tensor], state: Optional[Tensor], batch: int,
                      heads: int, fused: bool = True) -> Tensor:
    """``reference.decayed_attention``: ``[B * S, heads * vdim]`` in fp32."""
    if fused and _kn(q, k, v):
        from . import cuda_ops
        return cuda_ops.decayed_attention(q, k, v, decay, keep, state, batch, heads)
    o, final = ref.decayed_attention(q, k, v, decay, keep, state, batch, heads)
    if state is not None:
        state.copy_(final.detach())
    return o.reshape(q.size(0), -1)


def bonus_recurrence(r: Tensor, k: Tensor, v: Tensor, z: Tensor, w0: Tensor, u: Tensor, keep: Optional[Tensor],
                     state: Optional[Tensor], batch: int, heads: int, fused: bool = True) -> Tensor:
    """``reference.bonus_recurrence``: ``[B * S, heads * vdim]`` in fp32."""
    if fused and _kn(r, k, v, z, w0, u):
        from . import cuda_ops
        return cuda_ops.bonus_recurrence(r, k, v, z, w0, u, keep, state, batch, heads)
    o, final = ref.bonus_recurrence(r, k, v, z, w0, u, keep, state, batch, heads)
    if state is not None:
        state.copy_(final.detach())
    return o.reshape(r.size(0), -1)


def matrix_memory(q: Tensor, k: Tensor, v: Tensor, z: Tensor, bias: Tensor, cap: float, keep: Optional[Tensor],
                  state: Optional[Tensor], top: Optional[Tensor], batch: int, heads: int,
                  fused: bool = True) -> Tuple[Tensor, Tensor, Tensor]:
    """``reference.matrix_memory``: ``S^T q``, ``n . q`` and the running maximum of every token (fp32)."""
    if fused and _kn(q, k, v, z, bias):
        from . import cuda_ops
        return cuda_ops.matrix_memory(q, k, v, z, bias, cap, keep, state, top, batch, heads)
    o, nq, m, final, last = ref.matrix_memory(q, k, v, z, bias, cap, keep, state, top, batch, heads)
    if state is not None:
        state.copy_(final.detach())
        top.copy_(last.detach())
    return o, nq, m


def token_shift(h: Tensor, mu: Tensor, batch: int, keep: Optional[Tensor], prev: Optional[Tensor], fused: bool = True) -> Tensor:
    if fused and _kn(h, mu):
        from . import cuda_ops
        return cuda_ops.token_shift(h, mu, batch, keep, prev)
    mixed, last = ref.token_shift(h, mu, batch, keep, prev)
    if prev is not None:
        prev.copy_(last.detach())
    return mixed


def causal_conv(x: Tensor, w: Tensor, bias: Optional[Tensor], batch: int, keep: Optional[Tensor], prev: Optional[Tensor],
                silu: bool = False, residual: bool = False, fused: bool = True) -> Tensor:
    if fused and _kn(x, w, bias):
        from . import cuda_ops
        return cuda_ops.causal_conv(x, w, bias, batch, keep, prev, silu, residual)
    y, last = ref.causal_conv(x, w, bias, batch, keep, prev, silu, residual)
    if prev is not None:
        prev.copy_(last.detach())
    return y


def selective_scan(x: Tensor, dt: Tensor, dt_bias: Tensor, a_log: Tensor, b: Tensor, c: Tensor, d: Tensor, z: Tensor, batch: int,
                   keep: Optional[Tensor], state: Optional[Tensor], fused: bool = True) -> Tensor:
    if fused and _kn(x, dt, dt_bias, a_log, b, c, d, z):
        from . import cuda_ops
        return cuda_ops.selective_scan(x, dt, dt_bias, a_log, b, c, d, z, batch, keep, state)
    y, final = ref.selective_scan(x, dt, dt_bias, a_log, b, c, d, z, batch, keep, state)
    if state is not None:
        state.copy_(final.detach())
    return y
