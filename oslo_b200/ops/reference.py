"""Plain PyTorch statements of every op in this package.

They are the numerical oracle for the CUDA kernels and the execution path on CPU
(gloo ranks, unit tests). Semantics follow the eager model code of the reference
(attention: oslo/models/gptj/modeling_gptj.py:151-191, rotary :49-77; causal softmax:
oslo/fused_kernels/includes/fused_triang_softmax.h:134-251; padded softmax:
includes/fused_softmax.h:111-229; n-gram ban: fused_ngram_repeat_block.cu:18-49).
"""
from __future__ import annotations

import math
from typing import Optional, Tuple

import torch
import torch.nn.functional as F
from torch import Tensor


def gelu_tanh(x: Tensor) -> Tensor:
    return 0.5 * x * (1.0 + torch.tanh(0.7978845608028654 * (x + 0.044715 * x * x * x)))


def linear(x: Tensor, weight: Tensor, bias: Optional[Tensor] = None, reversed: bool = False,
           activation: Optional[str] = None) -> Tensor:
    """``x @ W.T`` (``nn.Linear`` layout) or ``x @ W`` when ``reversed`` (Conv1D ``[in, out]`` layout)."""
    y = torch.matmul(x, weight if reversed else weight.t())
    if bias is not None:
        y = y + bias
    if activation in ("gelu", "gelu_new", "gelu_tanh", "gelu_pytorch_tanh"):
        y = gelu_tanh(y)
    elif activation is not None:
        raise ValueError(f"unsupported fused activation {activation!r}")
    return y


def layer_norm(x: Tensor, weight: Tensor, bias: Optional[Tensor], eps: float) -> Tensor:
    return F.layer_norm(x, (x.size(-1),), weight, bias, eps)


def bias_gelu(x: Tensor, bias: Optional[Tensor]) -> Tensor:
    return gelu_tanh(x if bias is None else x + bias)


def bias_dropout_residual(x: Tensor, bias: Optional[Tensor], residual: Optional[Tensor], p: float,
                          training: bool) -> Tensor:
    y = x if bias is None else x + bias
    y = F.dropout(y, p=p, training=training)
    return y if residual is None else y + residual


def rotary_tables(positions: Tensor, rotary_dim: int, base: float = 10000.0) -> Tuple[Tensor, Tensor]:
    """sin/cos of shape ``[..., rotary_dim // 2]`` in fp32 for integer ``positions``."""
    inv = 1.0 / (base ** (torch.arange(0, rotary_dim, 2, device=positions.device, dtype=torch.float32) / rotary_dim))
    ang = positions.to(torch.float32).unsqueeze(-1) * inv
    return torch.sin(ang), torch.cos(ang)


def rotary_interleaved(x: Tensor, positions: Tensor, rotary_dim: int, base: float = 10000.0) -> Tensor:
    """GPT-J rotary embedding: pairs ``(x[2i], x[2i+1])`` of the first ``rotary_dim`` dims are rotated.

    ``x``: ``[B, S, heads, head_dim]``; ``positions``: ``[B, S]`` (or ``[S]``).
    """
    if positions.dim() == 1:
        positions = positions.unsqueeze(0).expand(x.size(0), -1)
    sin, cos = rotary_tables(positions, rotary_dim, base)  # [B, S, r/2]
    sin, cos = sin.unsqueeze(2), cos.unsqueeze(2)
    xr = x[..., :rotary_dim].to(torch.float32)
    x1, x2 = xr[..., 0::2], xr[..., 1::2]
    o1 = x1 * cos - x2 * sin
    o2 = x2 * cos + x1 * sin
    rot = torch.stack((o1, o2), dim=-1).flatten(-2)
    return torch.cat((rot.to(x.dtype), x[..., rotary_dim:]), dim=-1)


def attention_mask_bias(sq: int, sk: int, device, causal: bool, window: Optional[int]) -> Optional[Tensor]:
    """Boolean ``[sq, sk]`` keep-mask. Query ``i`` sits at absolute position ``sk - sq + i``."""
    if not causal and window is None:
        return None
    qpos = torch.arange(sk - sq, sk, device=device).unsqueeze(1)
    kpos = torch.arange(sk, device=device).unsqueeze(0)
    keep = torch.ones(sq, sk, dtype=torch.bool, device=device)
    if causal:
        keep &= kpos <= qpos
    if window is not None:
        keep &= kpos > qpos - window
    return keep


def attention(q: Tensor, k: Tensor, v: Tensor, causal: bool = True, window: Optional[int] = None,
              scale: Optional[float] = None, key_padding_mask: Optional[Tensor] = None,
              dropout_p: float = 0.0, training: bool = False, return_probs: bool = False):
    """Softmax attention on ``[B, heads, S, D]`` tensors, fp32 scores.

    ``key_padding_mask``: ``[B, Sk]`` with 1 = keep, 0 = padded key. ``window`` keeps keys
    ``q_pos - window < k_pos <= q_pos`` (GPT-Neo local attention).
    """
    sq, sk = q.size(-2), k.size(-2)
    if scale is None:
        scale = 1.0 / math.sqrt(q.size(-1))
    s = torch.matmul(q.to(torch.float32), k.to(torch.float32).transpose(-1, -2)) * scale
    keep = attention_mask_bias(sq, sk, q.device, causal, window)
    neg = torch.finfo(torch.float32).min
    if keep is not None:
        s = s.masked_fill(~keep, neg)
    if key_padding_mask is not None:
        s = s.masked_fill(~key_padding_mask.to(torch.bool)[:, None, None, :], neg)
    p = torch.softmax(s, dim=-1)
    if dropout_p > 0.0 and training:
        p = F.dropout(p, dropout_p, True)
    out = torch.matmul(p, v.to(torch.float32)).to(q.dtype)
    return (out, p) if return_probs else out


def scaled_upper_triang_masked_softmax(x: Tensor, scale: float) -> Tensor:
    """Causal softmax of ``scale * x`` on ``[batches, S, S]``; entries above the diagonal are exactly 0."""
    s = x.size(-1)
    keep = torch.ones(s, s, dtype=torch.bool, device=x.device).tril()
    y = (x.to(torch.float32) * scale).masked_fill(~keep, float("-inf"))
    return torch.softmax(y, dim=-1).to(x.dtype)


def scaled_masked_softmax(x: Tensor, mask: Tensor, scale: float) -> Tensor:
    """Softmax of ``scale * x`` on ``[b, heads, sq, sk]`` where ``mask`` (1 = masked) replaces by -10000."""
    y = x.to(torch.float32) * scale
    y = y.masked_fill(mask.to(torch.bool), -10000.0)
    return torch.softmax(y, dim=-1).to(x.dtype)


def softmax_backward(y: Tensor, dy: Tensor, scale: float) -> Tensor:
    yf, gf = y.to(torch.float32), dy.to(torch.float32)
    t = yf * gf
    return (scale * (t - yf * t.sum(-1, keepdim=True))).to(y.dtype)


def cross_entropy(logits: Tensor, labels: Tensor, ignore_index: int = -100) -> Tensor:
    """Mean token cross-entropy in fp32 over ``[N, V]`` logits."""
    return F.cross_entropy(logits.to(torch.float32), labels, ignore_index=ignore_index)


def adam_step(p32: Tensor, g: Tensor, m: Tensor, v: Tensor, step: int, lr: float, beta1: float, beta2: float,
              eps: float, weight_decay: float, grad_scale: float = 1.0, p_lp: Optional[Tensor] = None) -> None:
    """In-place AdamW on fp32 master weights; optionally refreshes a low-precision copy."""
    gf = g.to(torch.float32) * grad_scale
    m.mul_(beta1).add_(gf, alpha=1 - beta1)
    v.mul_(beta2).addcmul_(gf, gf, value=1 - beta2)
    bc1 = 1 - beta1 ** step
    bc2 = 1 - beta2 ** step
    if weight_decay != 0.0:
        p32.mul_(1 - lr * weight_decay)
    denom = (v / bc2).sqrt_().add_(eps)
    p32.addcdiv_(m / bc1, denom, value=-lr)
    if p_lp is not None:
        p_lp.copy_(p32)


def banned_ngram_tokens(tokens: Tensor, n: int):
    """For each row, tokens that would complete an n-gram already present in that row."""
    out = []
    rows = tokens.tolist()
    for row in rows:
        banned = set()
        if len(row) + 1 >= n:
            tail = tuple(row[len(row) - n + 1:]) if n > 1 else ()
            for i in range(len(row) - n + 1):
                if tuple(row[i:i + n - 1]) == tail:
                    banned.add(row[i + n - 1])
        out.append(sorted(banned))
    return out


def ban_repeated_ngrams(tokens: Tensor, lprobs: Tensor, n: int) -> Tensor:
    """Set ``lprobs[row, tok] = -inf`` for every token that would repeat an n-gram of ``tokens[row]``."""
    if n <= 0:
        return lprobs
    for r, banned in enumerate(banned_ngram_tokens(tokens, n)):
        if banned:
            lprobs[r, banned] = float("-inf")
    return lprobs


# ---------------------------------------------------------------------------------------------------------------
# RMS norms, gated residual joins, gated linear recurrence, latent attention with a sink, mixture of experts. All of them
# compute in fp32 and are differentiable; rows are tokens ([batch * positions, features]) unless stated otherwise.
def rms_norm(x: Tensor, w: Tensor, eps: float, offset: float = 0.0) -> Tensor:
    """``x / sqrt(mean(x^2) + eps) * (offset + w)`` over the last dim, in ``w``'s dtype (``offset=1``: the weight is stored
    around zero)."""
    xf = x.to(torch.float32)
    r = torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps)
    return (xf * r * (offset + w.to(torch.float32))).to(w.dtype)


def residual_join(x: Tensor, y: Tensor, gate: Tensor, gate_bias: Tensor, w_post: Tensor, w_next: Optional[Tensor],
                  eps: float, slots: Optional[Tensor] = None, slot_weights: Optional[Tensor] = None):
    """``x + norm(y * sigmoid(gate + gate_bias))`` in fp32, and the norm of that for the next sublayer (or ``None``). With
    ``slot_weights`` ``[tokens, top]`` the sublayer's result is the weighted sum of ``y``'s rows ``slots``
    (``token * top + choice`` when ``slots`` is ``None``)."""
    yf = y.to(torch.float32)
    if slot_weights is not None:
        n, top = slot_weights.shape
        picked = yf.view(n, top, -1) if slots is None else yf[slots.reshape(-1).to(torch.long)].view(n, top, -1)
        yf = (picked * slot_weights.unsqueeze(-1)).sum(1)
    z = yf * torch.sigmoid(gate.to(torch.float32) + gate_bias.to(torch.float32))
    r = torch.rsqrt(z.pow(2).mean(-1, keepdim=True) + eps)
    x = x + z * r * (1.0 + w_post.to(torch.float32))
    return x, (rms_norm(x, w_next, eps, 1.0) if w_next is not None else None)


def silu_mul(gate: Tensor, up: Tensor) -> Tensor:
    return F.silu(gate.to(torch.float32)).mul(up.to(torch.float32)).to(up.dtype)


def recurrence(q: Tensor, f: Tensor, v: Tensor, f_bias: Tensor, lower: Tensor, keep: Optional[Tensor],
               state: Optional[Tensor], batch: int, heads: int, dim: int, vdim: int) -> Tuple[Tensor, Tensor]:
    """Linear attention whose forget gate also decides what is written: per head and key channel
    ``1 - k = lower + (1 - lower) sigmoid(f + f_bias)``, ``S <- S + k (v - S)``, ``o = S^T silu(q)``.

    ``q``/``f`` ``[batch * S, heads * dim]``, ``v`` ``[batch * S, heads * vdim]``; ``keep`` ``[batch, S]`` (0: the token leaves
    the state alone and its output is 0); ``state`` ``[batch, heads, dim, vdim]`` fp32 or ``None`` (zero). Returns
    ``[batch, S, heads, vdim]`` in fp32 and the final state."""
    lo = lower.to(torch.float32)
    k = ((1.0 - lo) * torch.sigmoid(-(f.to(torch.float32) + f_bias.to(torch.float32)))).view(batch, -1, heads, dim)
    qs = F.silu(q.to(torch.float32)).view(batch, -1, heads, dim)
    vf = v.to(torch.float32).reshape(batch, -1, heads, vdim)
    if keep is not None:
        on = (keep != 0).to(torch.float32)[:, :, None, None]
        k, qs = k * on, qs * on
    s = torch.zeros(batch, heads, dim, vdim, dtype=torch.float32, device=q.device) if state is None else state
    out = []
    for t in range(k.size(1)):
        s = s + k[:, t].unsqueeze(-1) * (vf[:, t].unsqueeze(-2) - s)
        out.append(torch.einsum("bhi,bhij->bhj", qs[:, t], s))
    return torch.stack(out, dim=1), s


def sink_attention(q: Tensor, k: Tensor, v: Tensor, keep: Optional[Tensor], sink: Tensor, gate: Tensor, scale: float):
    """Causal softmax attention whose denominator also holds ``exp(sink[head])``; head ``h``'s output times
    ``sigmoid(gate[:, h])``. ``q`` ``[B, Sq, H, D]`` are the last positions of ``k``/``v`` ``[B, Sk, H, *]``; ``keep``
    ``[B, Sk]``; ``gate`` ``[B * Sq, H]``. Returns ``[B * Sq, H * Dv]`` and the weights ``[B, H, Sq, Sk]``."""
    b, sq, h, _ = q.shape
    sk = k.size(1)
    s = torch.einsum("bqhd,bkhd->bhqk", q.to(torch.float32), k.to(torch.float32)) * scale
    vis = attention_mask_bias(sq, sk, q.device, True, None)[None, None]
    if keep is not None:
        vis = vis & (keep != 0)[:, None, None, :]
    s = s.masked_fill(~vis, float("-inf"))
    s = torch.cat([s, sink.to(torch.float32)[None, :, None, None].expand(b, h, sq, 1)], dim=-1)
    p = torch.softmax(s, dim=-1)[..., :sk]
    o = torch.einsum("bhqk,bkhd->bqhd", p, v.to(torch.float32))
    o = o * torch.sigmoid(gate.to(torch.float32)).view(b, sq, h, 1)
    return o.reshape(b * sq, -1).to(q.dtype), p


def latent_decode(q: Tensor, w_uk: Tensor, w_uv: Tensor, cache: Tensor, lengths: Tensor, keep: Optional[Tensor],
                  sink: Tensor, gate: Tensor, scale: float, heads: int) -> Tensor:
    """One query per row over a cache of latents ``[B, T, rank]`` without expanding keys or values: the query takes
    ``W_uk``, the weighted sum of latents takes ``W_uv``. ``q`` ``[B, heads * dim]``; returns ``[B, heads * vdim]``."""
    b, t, r = cache.shape
    c = cache.to(torch.float32)
    qa = torch.einsum("bhd,hdr->bhr", q.to(torch.float32).view(b, heads, -1), w_uk.to(torch.float32).view(heads, -1, r)) * scale
    s = torch.einsum("bhr,btr->bht", qa, c)
    vis = torch.arange(t, device=q.device)[None, :] < lengths[:, None]
    if keep is not None:
        vis = vis.clone()
        n = min(t, keep.size(1))
        vis[:, :n] &= keep[:, :n] != 0
    s = s.masked_fill(~vis[:, None, :], float("-inf"))
    s = torch.cat([s, sink.to(torch.float32)[None, :, None].expand(b, heads, 1)], dim=-1)
    p = torch.softmax(s, dim=-1)[..., :t]
    o = torch.einsum("bhr,hvr->bhv", torch.einsum("bht,btr->bhr", p, c), w_uv.to(torch.float32).view(heads, -1, r))
    return (o * torch.sigmoid(gate.to(torch.float32)).unsqueeze(-1)).reshape(b, -1).to(q.dtype)


def moe_route(h: Tensor, w: Tensor, bias: Tensor, top: int) -> Tuple[Tensor, Tensor]:
    """The ``top`` experts with the largest ``W h + b`` per token (``[tokens, top]``, int32) and the softmax over those logits."""
    z = torch.matmul(h.to(torch.float32), w.to(torch.float32).t()) + bias.to(torch.float32)
    picked, idx = torch.topk(z, top, dim=-1)
    return idx.to(torch.int32), torch.softmax(picked, dim=-1)


def moe_experts(h: Tensor, idx: Tensor, up: Tensor, down: Tensor) -> Tensor:
    """``W_down relu(W_up h)^2`` of every (token, choice): ``[tokens * top, width]``; ``up`` ``[experts, ff, width]``,
    ``down`` ``[experts, width, ff]``."""
    n, top = idx.shape
    flat = idx.reshape(-1).to(torch.long)
    rows = h.repeat_interleave(top, dim=0)
    out = h.new_zeros(n * top, down.size(1))
    for e in flat.unique().tolist():
        at = (flat == e).nonzero(as_tuple=True)[0]
        a = torch.relu(torch.matmul(rows[at], up[e].t())).pow(2)
        out = out.index_copy(0, at, torch.matmul(a, down[e].t()).to(out.dtype))
    return out
