"""Plain PyTorch statements of every op in this package.

They are the numerical oracle for the CUDA kernels and the execution path on CPU
(gloo ranks, unit tests). Semantics follow the eager model code of the reference
(attention: oslo/models/gptj/modeling_gptj.py:151-191, rotary :49-77; causal softmax:
oslo/fused_kernels/includes/fused_triang_softmax.h:134-251; padded softmax:
includes/fused_softmax.h:111-229; n-gram ban: fused_ngram_repeat_block.cu:18-49).
"""
from __future__ import annotations

import math
from typing import Dict, NamedTuple, Optional, Tuple

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
    elif activation == "relu2":
        y = torch.relu(y).pow(2)
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


def visible_keys(qpos: Tensor, kpos: Tensor, window: int, keep_first: int, lead: Optional[Tensor]) -> Tensor:
    """Which of the columns ``kpos`` a query at column ``qpos`` may read (both broadcast; ``lead`` has the shape of a batch of them):
    those up to its own, with a ``window`` > 0 only the last ``window`` of them and the sequence's first ``keep_first``, whose
    columns start behind ``lead`` columns of padding."""
    vis = kpos <= qpos
    if window > 0:
        near = qpos - kpos < window
        if keep_first > 0:
            near = near | ((kpos if lead is None else kpos - lead) < keep_first)
        vis = vis & near
    return vis


def output_gate(o: Tensor, gate: Optional[Tensor]) -> Tensor:
    """``o`` ``[rows, heads, vdim]`` times the sigmoid of ``gate`` ``[rows, heads]`` (one factor per head) or ``[rows, heads * vdim]``."""
    if gate is None:
        return o
    g = torch.sigmoid(gate.to(torch.float32))
    return o * (g.unsqueeze(-1) if g.size(-1) == o.size(1) else g.view(o.shape))


def sink_attention(q: Tensor, k: Tensor, v: Tensor, keep: Optional[Tensor], sink: Optional[Tensor], gate: Optional[Tensor],
                   scale: float, softcap: float = 0.0, window: int = 0, keep_first: int = 0, lead: Optional[Tensor] = None,
                   q_rot: Optional[Tensor] = None, k_rot: Optional[Tensor] = None):
    """Causal softmax attention; with ``sink`` the denominator also holds ``exp(sink[head])``; with ``gate`` ``[B * Sq, H]`` or
    ``[B * Sq, H * Dv]`` the output is multiplied by its sigmoid, with ``softcap`` scores become ``softcap * tanh(score / softcap)``.
    ``q`` ``[B, Sq, H, D]`` are the last positions of ``k``/``v`` ``[B, Sk, G, *]``; query head ``h`` reads key head ``h // (H / G)``
    (keys and values may differ in ``G``); ``keep`` ``[B, Sk]``; ``window``, ``keep_first``, ``lead`` ``[B]``: ``visible_keys``. ``q_rot`` ``[B, Sq, H, R]`` and ``k_rot`` ``[B, Sk,
    R]``, a part of the keys that all heads share, add ``q_rot . k_rot`` to the scores before the scale. Returns ``[B * Sq, H * Dv]``
    and the weights ``[B, H, Sq, Sk]``."""
    b, sq, h, _ = q.shape
    sk = k.size(1)
    k, v = (t if t.size(2) == h else t.repeat_interleave(h // t.size(2), dim=2) for t in (k, v))
    s = torch.einsum("bqhd,bkhd->bhqk", q.to(torch.float32), k.to(torch.float32))
    if q_rot is not None:
        s = s + torch.einsum("bqhd,bkd->bhqk", q_rot.to(torch.float32), k_rot.to(torch.float32))
    s = s * scale
    if softcap:
        s = softcap * torch.tanh(s / softcap)
    qpos = torch.arange(sk - sq, sk, device=q.device)[None, None, :, None]
    kpos = torch.arange(sk, device=q.device)[None, None, None, :]
    vis = visible_keys(qpos, kpos, window, keep_first, None if lead is None else lead.view(-1, 1, 1, 1))
    if keep is not None:
        vis = vis & (keep != 0)[:, None, None, :]
    s = s.masked_fill(~vis, float("-inf"))
    if sink is not None:
        s = torch.cat([s, sink.to(torch.float32)[None, :, None, None].expand(b, h, sq, 1)], dim=-1)
        p = torch.softmax(s, dim=-1)[..., :sk]
    else:
        some = vis.any(-1, keepdim=True)               # a padded query may see nothing: its row is zero
        p = torch.softmax(s.masked_fill(~some, 0.0), dim=-1) * some
    o = torch.einsum("bhqk,bkhd->bqhd", p, v.to(torch.float32))
    o = output_gate(o.reshape(b * sq, h, -1), gate)
    return o.reshape(b * sq, -1).to(q.dtype), p


def rotate_halves(x: Tensor, positions: Tensor, freq: Tensor) -> Tensor:
    """``x`` ``[B, S, heads, 2 n]``: dim ``i`` and dim ``i + n`` turn by ``positions * freq[i]`` (fp32); ``positions`` ``[B, S]``."""
    n = freq.numel()
    xf = x.to(torch.float32)
    ang = (positions.to(torch.float32).unsqueeze(-1) * freq).unsqueeze(2)
    sin, cos = torch.sin(ang), torch.cos(ang)
    a, b = xf[..., :n], xf[..., n:]
    return torch.cat((a * cos - b * sin, b * cos + a * sin), dim=-1).to(x.dtype)


def latent_decode(q: Tensor, w_uk: Tensor, w_uv: Tensor, cache: Tensor, lengths: Tensor, keep: Optional[Tensor],
                  sink: Optional[Tensor], gate: Tensor, scale: float, heads: int, positions: Optional[Tensor] = None,
                  freq: Optional[Tensor] = None) -> Tensor:
    """One query per row over a cache of latents ``[B, T, rank + rot]`` without expanding keys or values: the query takes
    ``W_uk``, the weighted sum of latents takes ``W_uv``. ``q`` ``[B, heads * (dim + rot)]``; the last ``rot`` = ``2 * len(freq)`` dims of a
    head are rotated (``rotate_halves``) by ``positions`` ``[B, 1]`` and meet the last ``rot`` of a cached row. Returns ``[B, heads *
    vdim]``."""
    b, t, _ = cache.shape
    r = w_uk.size(1)
    rot = cache.size(2) - r
    c = cache.to(torch.float32)
    qh = q.to(torch.float32).view(b, heads, -1)
    dim = qh.size(-1) - rot
    qa = torch.einsum("bhd,hdr->bhr", qh[..., :dim], w_uk.to(torch.float32).view(heads, dim, r))
    if rot:
        qa = torch.cat([qa, rotate_halves(qh[..., dim:].unsqueeze(1), positions, freq)[:, 0]], dim=-1)
    s = torch.einsum("bhr,btr->bht", qa * scale, c)
    vis = torch.arange(t, device=q.device)[None, :] < lengths[:, None]
    if keep is not None:
        vis = vis.clone()
        n = min(t, keep.size(1))
        vis[:, :n] &= keep[:, :n] != 0
    s = s.masked_fill(~vis[:, None, :], float("-inf"))
    if sink is not None:
        s = torch.cat([s, sink.to(torch.float32)[None, :, None].expand(b, heads, 1)], dim=-1)
    p = torch.softmax(s, dim=-1)[..., :t]
    o = torch.einsum("bhr,hvr->bhv", torch.einsum("bht,btr->bhr", p, c[..., :r]), w_uv.to(torch.float32).view(heads, -1, r))
    return output_gate(o, gate).reshape(b, -1).to(q.dtype)


def moe_route(h: Tensor, w: Tensor, bias: Optional[Tensor], top: int, scored=False) -> Tuple[Tensor, Tensor]:
    """The ``top`` experts with the largest ``W h + b`` per token (``[tokens, top]``, int32) and the softmax over those logits.
    ``scored``: scores are the softmax of ``W h`` over all experts, the largest ``score + b`` are chosen, and the weights are the
    chosen scores without ``b``, divided by their sum. ``scored="sigmoid"``: the largest ``W h`` are chosen (no ``b``), their weights are
    ``sigmoid(W h)``."""
    z = torch.matmul(h.to(torch.float32), w.to(torch.float32).t())
    if scored == "sigmoid":
        picked, idx = torch.topk(z, top, dim=-1)
        return idx.to(torch.int32), torch.sigmoid(picked)
    if scored:
        score = torch.softmax(z, dim=-1)
        idx = torch.topk(score + bias.to(torch.float32), top, dim=-1).indices
        picked = score.gather(-1, idx)
        return idx.to(torch.int32), picked / (picked.sum(-1, keepdim=True) + 1e-20)
    picked, idx = torch.topk(z + bias.to(torch.float32), top, dim=-1)
    return idx.to(torch.int32), torch.softmax(picked, dim=-1)


def moe_experts(h: Tensor, idx: Tensor, up: Tensor, down: Tensor, unit: str = "relu2", limit: float = 0.0, alpha: float = 1.702,
                scale: Optional[Tensor] = None) -> Tensor:
    """Every (token, choice): ``[tokens * top, width]``; ``down`` ``[experts, width, ff]``. ``unit`` ``"relu2"``: ``W_down relu(W_up h)^2``
    with ``up`` ``[experts, ff, width]``; ``"silu"``: ``W_down (silu(W_gate h) * W_up h)`` with ``up`` ``[experts, 2 ff, width]``, rows of the
    two matrices in turns; ``"clamped"``: the same with ``clamped_glu(limit, alpha)`` for ``silu``. ``scale`` ``[tokens, top]`` multiplies what
    an expert reads. Rows of choices that are no expert (``idx >= experts``) are zeros."""
    n, top = idx.shape
    flat = idx.reshape(-1).to(torch.long)
    rows = h.repeat_interleave(top, dim=0)
    if scale is not None:
        rows = (rows.to(torch.float32) * scale.reshape(-1, 1)).to(h.dtype)
    out = h.new_zeros(n * top, down.size(1))
    for e in flat.unique().tolist():
        if e >= up.size(0):
            continue
        at = (flat == e).nonzero(as_tuple=True)[0]
        a = torch.matmul(rows[at], up[e].t())
        if unit == "relu2":
            a = torch.relu(a).pow(2)
        elif unit == "clamped":
            a = clamped_glu(a[:, 0::2], a[:, 1::2], limit, alpha)
        else:
            a = silu_mul(a[:, 0::2], a[:, 1::2])
        out = out.index_copy(0, at, torch.matmul(a, down[e].t()).to(out.dtype))
    return out


# ---------------------------------------------------------------------------------------------------------------
# Hyper-connections: several residual streams, mixed by every sublayer.
class SublayerResult(NamedTuple):
    """What a sublayer hands to ``hyper_join``: ``y`` ``[tokens, width]``, or with ``weights`` ``[tokens, top]`` the weighted sum of
    ``y``'s rows ``slots`` (``token * top + choice`` when ``None``), where a choice ``>= experts`` stands for the sublayer's input ``h``
    itself; plus ``sigmoid(shared_gate) * shared`` (``shared_gate`` ``[tokens, 1]``) when there is a ``shared``."""
    y: Tensor
    slots: Optional[Tensor] = None
    weights: Optional[Tensor] = None
    choice: Optional[Tensor] = None
    experts: int = 0
    h: Optional[Tensor] = None
    shared: Optional[Tensor] = None
    shared_gate: Optional[Tensor] = None


def collect_result(r: SublayerResult) -> Tensor:
    """The sublayer's result as fp32 rows ``[tokens, width]``."""
    y = r.y.to(torch.float32)
    if r.weights is not None:
        n, top = r.weights.shape
        if r.choice is not None:
            own = (r.choice.to(torch.long) < r.experts)
        slots = torch.arange(n * top, device=y.device).view(n, top) if r.slots is None else r.slots.to(torch.long)
        if r.choice is None:
            picked = y[slots]
        else:
            picked = torch.where(own.unsqueeze(-1), y[torch.where(own, slots, torch.zeros_like(slots))], r.h.to(torch.float32).unsqueeze(1))
        y = (picked * r.weights.unsqueeze(-1)).sum(1)
    if r.shared is not None:
        y = y + torch.sigmoid(r.shared_gate.to(torch.float32)) * r.shared.to(torch.float32)
    return y


def hyper_join(x: Tensor, result: Optional[SublayerResult], w_out: Optional[Tensor], mix: Optional[Tensor], w_in: Optional[Tensor],
               w_norm: Tensor, eps: float, scale: float = 1.0) -> Tuple[Tensor, Tensor]:
    """Streams ``x`` ``[tokens, streams, width]`` (fp32) take a sublayer's result ``y``: ``x_t <- sum_s mix[s, t] x_s + w_out[t] y`` (all
    streams from the old ones; no ``result``: they stay), and what the next sublayer reads: ``u = sum_t w_in[t] x_t`` (``None``: their
    plain sum), normed with weight ``1 + w_norm`` and multiplied by ``scale``."""
    if result is not None:
        y = collect_result(result)
        x = torch.einsum("nsw,st->ntw", x, mix.to(torch.float32)) + w_out.to(torch.float32)[None, :, None] * y.unsqueeze(1)
    u = x.sum(1) if w_in is None else (x * w_in.to(torch.float32)[None, :, None]).sum(1)
    r = torch.rsqrt(u.pow(2).mean(-1, keepdim=True) + eps)
    return x, (u * r * ((1.0 + w_norm.to(torch.float32)) * scale)).to(w_norm.dtype)


# ---------------------------------------------------------------------------------------------------------------
# Residual joins of parallel branches, grouped-query attention, linear recurrences with decays of their own, token shift,
# causal convolution, selective scan, clamped gated units.
class Branch(NamedTuple):
    """A result on its way to the residual stream: ``factor * y``, with a ``weight`` ``[width]`` ``factor * norm(y) * weight``, or
    (``normed=False``) ``factor * y * weight``. With ``top`` > 0 a token's ``y`` is the sum of ``top`` rows: those that ``slots`` ``[rows,
    top]`` names, or (``None``) rows ``top * token`` and on."""
    y: Tensor                              # [rows, width], or more rows with ``top``
    weight: Optional[Tensor] = None
    factor: float = 1.0
    normed: bool = True
    slots: Optional[Tensor] = None
    top: int = 0


def branch_join(x: Tensor, branches, mult: float, eps: float, w_next, copy: Optional[torch.dtype] = None) -> Tuple[Tensor, list]:
    """``x + mult`` times the sum of the ``branches`` (``Branch``) in fp32, and the RMS norms of that with every weight of ``w_next``
    (``[width]``, or one number). ``copy`` (without ``w_next``): instead of norms the sum itself in that dtype."""
    total = None
    for b in branches:
        b = Branch(*b)
        yf = b.y.to(torch.float32)
        if b.top:
            yf = (yf if b.slots is None else yf[b.slots.reshape(-1).to(torch.long)]).view(x.size(0), b.top, -1).sum(1)
        if b.weight is not None:
            if b.normed:
                yf = yf * torch.rsqrt(yf.pow(2).mean(-1, keepdim=True) + eps)
            yf = yf * b.weight.to(torch.float32)
        yf = yf if b.factor == 1.0 else yf * b.factor
        total = yf if total is None else total + yf
    if total is not None:
        x = x + mult * total
    return x, [x.to(copy)] if copy is not None else [rms_norm(x, w, eps) for w in w_next]


def token_gate(z: Tensor, ids: Tensor, table: Tensor, first: int) -> Tensor:
    """``gelu_tanh(z)`` times the columns ``first`` and on of the tokens' rows of ``table`` ``[vocab, *]``: ``z`` ``[rows, dim]``, ``ids``
    ``[rows]``."""
    e = table[ids.reshape(-1), first:first + z.size(1)]
    return (gelu_tanh(z.to(torch.float32)) * e.to(torch.float32)).to(z.dtype)


def clamped_glu(gate: Tensor, up: Tensor, limit: float, alpha: float) -> Tensor:
    """``g sigmoid(alpha g) (u + 1)`` with ``g = min(gate, limit)``, ``u = clamp(up, -limit, limit)``."""
    g = gate.to(torch.float32).clamp(max=limit)
    u = up.to(torch.float32).clamp(-limit, limit)
    return (g * torch.sigmoid(alpha * g) * (u + 1.0)).to(up.dtype)


def rotary_frequencies(rot_dims: int, base: float, scaling: Optional[Dict[str, float]] = None):
    """``base^(-2i / rot_dims)`` for the pairs of the rotated dims, as 32-bit floats rounded once. ``scaling`` (YaRN): pairs that turn
    less than ``slow`` times over ``original`` positions are slowed down by ``factor``, those that turn more than ``fast`` times keep
    their frequency, with a linear ramp in between."""
    freq = [base ** (-2.0 * i / rot_dims) for i in range(rot_dims // 2)]
    if scaling is None:
        return freq
    factor, original = float(scaling["factor"]), float(scaling["original"])
    pair = lambda turns: rot_dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))   # noqa: E731
    lo = max(math.floor(pair(float(scaling["fast"]))), 0)
    hi = min(math.ceil(pair(float(scaling["slow"]))), rot_dims - 1)
    ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(len(freq))]
    return [f / factor * r + f * (1.0 - r) for f, r in zip(freq, ramp)]


def rotary_amplitude(scaling: Optional[Dict[str, float]] = None) -> float:
    """What YaRN multiplies sines and cosines by."""
    return 1.0 if scaling is None else 0.1 * math.log(float(scaling["factor"])) + 1.0


def norm_rotate(x: Tensor, w: Optional[Tensor], eps: float, positions: Tensor, freq: Optional[Tensor], halves: bool = False,
                amplitude: float = 1.0) -> Tensor:
    """Per head of ``x`` ``[B, S, heads, D]``: RMS norm with weight ``w`` ``[D]`` (shared by the heads; ``None``: without a weight, and
    then before or after the rotation is the same), then the rotation of the first ``2 * len(freq)`` dims by ``positions * freq``
    (fp32), interleaved pairs or (``halves``) dim ``i`` with dim ``i + len(freq)``, sines and cosines times ``amplitude``; ``positions``
    ``[B, S]``."""
    return _norm_rotate(x, w, eps, positions, freq, halves, amplitude).to(x.dtype)


def _norm_rotate(x, w, eps, positions, freq, halves, amplitude) -> Tensor:
    y = x.to(torch.float32)
    y = y * torch.rsqrt(y.pow(2).mean(-1, keepdim=True) + eps)
    if w is not None:
        y = y * w.to(torch.float32)
    if freq is not None and freq.numel():
        r = 2 * freq.numel()
        ang = (positions.to(torch.float32).unsqueeze(-1) * freq).unsqueeze(2)
        sin, cos = amplitude * torch.sin(ang), amplitude * torch.cos(ang)
        a, b = (y[..., :r // 2], y[..., r // 2:r]) if halves else (y[..., :r:2], y[..., 1:r:2])
        turned = (a * cos - b * sin, b * cos + a * sin)
        y = torch.cat((*(turned if halves else (torch.stack(turned, dim=-1).flatten(-2),)), y[..., r:]), dim=-1)
    return y


def norm_rotate_fold(q: Tensor, w: Optional[Tensor], eps: float, positions: Tensor, freq: Optional[Tensor], talk: Tensor, groups: int,
                     halves: bool = False, amplitude: float = 1.0) -> Tensor:
    """Queries of attention whose heads' scores are mixed before the softmax (talking heads), ``score_h <- sum_g talk[h, g] score_g``,
    with ``groups`` key heads: since head ``g`` reads key head ``g // (H / groups)``, the mixed score is one product of the keys of
    all key heads together with the query ``[sum over the heads g of key head 0 of talk[h, g] q_g | the same of key head 1 | ...]``.
    Returns that, ``[B, S, H, groups * D]``, for ``q`` ``[B, S, H, D]``, normed and rotated first (``norm_rotate``; rounded once)."""
    b, s, h, d = q.shape
    y = _norm_rotate(q, w, eps, positions, freq, halves, amplitude).view(b, s, groups, h // groups, d)
    t = talk.to(torch.float32).view(h, groups, h // groups)
    return torch.einsum("hgr,bsgrd->bshgd", t, y).reshape(b, s, h, groups * d).to(q.dtype)


def grouped_decode(q: Tensor, k: Tensor, v: Tensor, lengths: Tensor, keep: Optional[Tensor], sink: Optional[Tensor], scale: float,
                   softcap: float = 0.0, gate: Optional[Tensor] = None, window: int = 0, keep_first: int = 0,
                   lead: Optional[Tensor] = None) -> Tensor:
    """One query per row: ``q`` ``[B, H, D]`` over caches ``[B, G, T, *]`` of which the first ``lengths[b]`` positions count;
    ``keep`` ``[B, <= T]``. Sink, gate ``[B, H]`` or ``[B, H * Dv]`` and window as in ``sink_attention``; keys and values may differ in
    ``G``. Returns ``[B, H * Dv]``."""
    b, h, _ = q.shape
    g, t = v.size(1), k.size(2)
    if k.size(1) != g:
        k = k.repeat_interleave(h // k.size(1), dim=1).view(b, g, h // g, t, -1)
    else:
        k = k.unsqueeze(2)
    at = torch.arange(t, device=q.device)[None, :]
    vis = visible_keys(lengths[:, None] - 1, at, window, keep_first, None if lead is None else lead[:, None])
    if keep is not None:
        n = min(t, keep.size(1))
        vis[:, :n] &= keep[:, :n] != 0
    qg = q.to(torch.float32).view(b, g, h // g, -1)
    s = torch.matmul(k.to(torch.float32), qg.unsqueeze(-1)).squeeze(-1) * scale
    if softcap:
        s = softcap * torch.tanh(s / softcap)
    s = s.masked_fill(~vis[:, None, None, :], float("-inf"))
    if sink is not None:
        s = torch.cat([s, sink.to(torch.float32).view(1, g, h // g, 1).expand(b, g, h // g, 1)], dim=-1)
    p = torch.softmax(s, dim=-1)[..., :t]
    # positions beyond the length may hold anything
    vf = torch.where(vis[:, None, :, None], v.to(torch.float32), torch.zeros((), device=v.device))
    o = torch.einsum("bgrt,bgtd->bgrd", p, vf).reshape(b, h, -1)
    return output_gate(o, gate).reshape(b, -1).to(q.dtype)


def gated_rms_norm(o: Tensor, w: Tensor, gate: Tensor, eps: float, group: int, act: str,
                   normalizer: Optional[Tuple[Tensor, Tensor]] = None) -> Tensor:
    """Every run of ``group`` columns of ``o`` ``[rows, n]`` divided by its root mean square, times ``w`` ``[n]``, times
    ``sigmoid(gate)`` or ``silu(gate)`` (``act``); in ``w``'s dtype. ``normalizer`` ``(z, m)``, both ``[rows, n / group]``: the runs are first
    divided by ``max(|z|, exp(-m)) + 1e-6``."""
    of = o.to(torch.float32).reshape(o.size(0), -1, group)
    if normalizer is not None:
        z, m = (t.reshape(o.size(0), -1, 1) for t in normalizer)
        of = of / (torch.maximum(z.abs(), torch.exp(-m)) + 1e-6)
    of = (of * torch.rsqrt(of.pow(2).mean(-1, keepdim=True) + eps)).view(o.size(0), -1)
    g = gate.to(torch.float32)
    g = torch.sigmoid(g) if act == "sigmoid" else F.silu(g)
    return (of * w.to(torch.float32) * g).to(w.dtype)


def memory_state_width(vdim: int) -> int:
    """Columns of a matrix-memory state: ``vdim`` values, the normaliser, and padding to a multiple of 4."""
    return (vdim + 1 + 3) // 4 * 4


def matrix_memory(q: Tensor, k: Tensor, v: Tensor, z: Tensor, bias: Tensor, cap: float, keep: Optional[Tensor], state: Optional[Tensor],
                  top: Optional[Tensor], batch: int, heads: int):
    """Linear attention with one input and one forget gate per head and token in the exponent (mLSTM). ``z`` ``[B * S, 2 * heads]`` and
    ``bias`` ``[2 * heads]``, input gates first: ``i = cap tanh((z_i + b_i) / cap)``, ``f = log sigmoid(cap tanh((z_f + b_f) / cap))``. With
    the running maximum ``m = max(f + m', i)`` (``m' = 0`` before the first token): ``S <- exp(f + m' - m) S + exp(i - m) k v^T``, ``n``
    likewise from ``k`` alone. ``q`` is scaled by ``dim^-1/2``. ``state`` ``[B, heads, dim, memory_state_width(vdim)]`` holds ``S`` and, in
    column ``vdim``, ``n``; ``top`` ``[B, heads]`` holds ``m``. A padded token leaves all of it as it is.
    Returns ``S^T q`` ``[B * S, heads * vdim]``, ``n . q`` and ``m`` ``[B * S, heads]`` (fp32), the final state and maximum."""
    dim, vdim = q.size(1) // heads, v.size(1) // heads
    qf, kf, vf = (t.to(torch.float32).reshape(batch, -1, heads, t.size(1) // heads) for t in (q, k, v))
    qf = qf * dim ** -0.5
    g = cap * torch.tanh((z.to(torch.float32) + bias.to(torch.float32)) / cap)
    i, f = g[:, :heads].reshape(batch, -1, heads), F.logsigmoid(g[:, heads:]).reshape(batch, -1, heads)
    v1 = F.pad(torch.cat([vf, torch.ones_like(vf[..., :1])], dim=-1), (0, memory_state_width(vdim) - vdim - 1))
    s = torch.zeros(batch, heads, dim, v1.size(-1), device=q.device) if state is None else state
    m = torch.zeros(batch, heads, device=q.device) if top is None else top
    out, tops = [], []
    for t in range(qf.size(1)):
        new_m = torch.maximum(f[:, t] + m, i[:, t])
        forget, write = torch.exp(f[:, t] + m - new_m), torch.exp(i[:, t] - new_m)
        new = forget[..., None, None] * s + (write[..., None] * kf[:, t]).unsqueeze(-1) * v1[:, t].unsqueeze(-2)
        on = None if keep is None else keep[:, t] != 0
        s = new if on is None else torch.where(on.view(-1, 1, 1, 1), new, s)
        m = new_m if on is None else torch.where(on.view(-1, 1), new_m, m)
        o = torch.einsum("bhi,bhij->bhj", qf[:, t], s)
        out.append(o if on is None else o * on.to(torch.float32).view(-1, 1, 1))
        tops.append(m)
    o = torch.stack(out, dim=1).reshape(q.size(0), heads, -1)
    return o[..., :vdim].reshape(q.size(0), heads * vdim), o[..., vdim], torch.stack(tops, dim=1).reshape(q.size(0), heads), s, m


def decayed_attention(q: Tensor, k: Tensor, v: Tensor, decay: Tensor, keep: Optional[Tensor], state: Optional[Tensor],
                      batch: int, heads: int) -> Tuple[Tensor, Tensor]:
    """Linear attention with one constant decay per head: ``S <- decay S + silu(k) silu(v)^T``, ``o = S^T silu(q)``. ``q``, ``k``
    ``[B * S, heads * dim]``, ``v`` ``[B * S, heads * vdim]``; ``keep`` ``[B, S]``: a padded token leaves the state as it is.
    Returns ``o`` ``[B, S, heads, vdim]`` (fp32) and the final state ``[B, heads, dim, vdim]``."""
    qf, kf, vf = (F.silu(t.to(torch.float32)).view(batch, -1, heads, t.size(1) // heads) for t in (q, k, v))
    s = torch.zeros(batch, heads, kf.size(-1), vf.size(-1), device=q.device) if state is None else state
    dec = decay.to(torch.float32).view(1, heads, 1, 1)
    out = []
    for t in range(kf.size(1)):
        new = dec * s + kf[:, t].unsqueeze(-1) * vf[:, t].unsqueeze(-2)
        s = new if keep is None else torch.where((keep[:, t] != 0).view(-1, 1, 1, 1), new, s)
        out.append(torch.einsum("bhi,bhij->bhj", qf[:, t], s))
    o = torch.stack(out, dim=1)
    return (o if keep is None else o * (keep != 0).to(torch.float32)[:, :, None, None]), s


def bonus_recurrence(r: Tensor, k: Tensor, v: Tensor, z: Tensor, w0: Tensor, u: Tensor, keep: Optional[Tensor],
                     state: Optional[Tensor], batch: int, heads: int) -> Tuple[Tensor, Tensor]:
    """Linear attention with a decay per token, head and key channel, ``w = exp(-exp(z + w0))``: a token reads the state before it
    and itself with a bonus, ``o = S^T r + (r . (u k)) v``, then ``S <- diag(w) S + k v^T``. ``r``, ``k``, ``z`` ``[B * S, heads *
    dim]``, ``v`` ``[B * S, heads * vdim]``, ``w0``, ``u`` ``[heads * dim]``. Returns as ``decayed_attention``."""
    rf, kf, vf = (t.to(torch.float32).view(batch, -1, heads, t.size(1) // heads) for t in (r, k, v))
    w = torch.exp(-torch.exp(z.to(torch.float32) + w0.to(torch.float32))).view(kf.shape)
    s = torch.zeros(batch, heads, kf.size(-1), vf.size(-1), device=r.device) if state is None else state
    bonus = (rf * u.to(torch.float32).view(heads, -1) * kf).sum(-1, keepdim=True) * vf
    out = []
    for t in range(kf.size(1)):
        out.append(torch.einsum("bhi,bhij->bhj", rf[:, t], s) + bonus[:, t])
        new = w[:, t].unsqueeze(-1) * s + kf[:, t].unsqueeze(-1) * vf[:, t].unsqueeze(-2)
        s = new if keep is None else torch.where((keep[:, t] != 0).view(-1, 1, 1, 1), new, s)
    o = torch.stack(out, dim=1)
    return (o if keep is None else o * (keep != 0).to(torch.float32)[:, :, None, None]), s


def token_shift(h: Tensor, mu: Tensor, batch: int, keep: Optional[Tensor], prev: Optional[Tensor]) -> Tuple[Tensor, Tensor]:
    """``h + (h' - h) mu[i]`` for every row of ``mu`` ``[P, width]``, with ``h'`` the row of the token before (``prev`` ``[B, width]``
    before the first one; zeros at the start of a sequence and after padding). Returns ``[P, B * S, width]`` and the last rows."""
    hb = h.view(batch, -1, h.size(-1)).to(torch.float32)
    if keep is not None:
        hb = hb * (keep != 0).to(torch.float32).unsqueeze(-1)
    first = torch.zeros_like(hb[:, 0]) if prev is None else prev
    before = torch.cat([first.unsqueeze(1), hb[:, :-1]], dim=1)
    m = mu.to(torch.float32).view(mu.size(0), 1, 1, -1)
    return (hb + (before - hb) * m).to(h.dtype).view(mu.size(0), h.size(0), -1), hb[:, -1]


def causal_conv(x: Tensor, w: Tensor, bias: Optional[Tensor], batch: int, keep: Optional[Tensor], prev: Optional[Tensor],
                silu: bool = False, residual: bool = False) -> Tuple[Tensor, Tensor]:
    """A causal convolution per channel: ``x`` ``[B * S, C]``, ``w`` ``[C, taps]`` with the current token's tap last, ``prev`` ``[B, taps -
    1, C]`` the inputs before (zeros when ``None``). ``silu``: of the result; ``residual``: the input is added to it. Returns the
    result and the last ``taps - 1`` inputs."""
    taps = w.size(1)
    xb = x.view(batch, -1, x.size(-1)).to(torch.float32)
    if keep is not None:
        xb = xb * (keep != 0).to(torch.float32).unsqueeze(-1)
    s = xb.size(1)
    head = xb.new_zeros(batch, taps - 1, xb.size(-1)) if prev is None else prev
    full = torch.cat([head, xb], dim=1)
    y = sum(w[:, j].to(torch.float32) * full[:, j:j + s] for j in range(taps))
    if bias is not None:
        y = bias.to(torch.float32) + y
    y = F.silu(y) if silu else y
    return (y + xb if residual else y).to(x.dtype).reshape(x.shape), full[:, s:]


def selective_scan(x: Tensor, dt: Tensor, dt_bias: Tensor, a_log: Tensor, b: Tensor, c: Tensor, d: Tensor, z: Tensor, batch: int,
                   keep: Optional[Tensor], state: Optional[Tensor]) -> Tuple[Tensor, Tensor]:
    """Per channel ``i`` and state ``n``: ``S <- exp(t A) S + t x B_n`` with the step ``t = softplus(dt + dt_bias)`` and ``A =
    -exp(a_log)``; ``y = sum_n S C_n + d x``, times ``silu(z)``. ``x``, ``dt``, ``z`` ``[B * S, C]``, ``b``, ``c`` ``[B * S, N]``,
    ``a_log`` ``[C, N]``. A padded token leaves the state as it is. Returns ``[B * S, C]`` and the state ``[B, C, N]``."""
    step = F.softplus(dt.to(torch.float32) + dt_bias.to(torch.float32), threshold=30.0).view(batch, -1, x.size(-1))
    if keep is not None:
        step = step * (keep != 0).to(torch.float32).unsqueeze(-1)
    a = -torch.exp(a_log.to(torch.float32))
    xf = x.to(torch.float32).view(step.shape)
    bf, cf = (t.to(torch.float32).view(batch, -1, t.size(-1)) for t in (b, c))
    s = torch.zeros(batch, *a_log.shape, device=x.device) if state is None else state
    out = []
    for t in range(step.size(1)):
        s = torch.exp(step[:, t].unsqueeze(-1) * a) * s + (step[:, t] * xf[:, t]).unsqueeze(-1) * bf[:, t].unsqueeze(1)
        out.append(torch.einsum("bcn,bn->bc", s, cf[:, t]))
    y = torch.stack(out, dim=1) + d.to(torch.float32) * xf
    return (y.reshape(x.shape) * F.silu(z.to(torch.float32))).to(x.dtype), s
