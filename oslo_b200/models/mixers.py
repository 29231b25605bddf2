"""Token mixers and feed-forwards that are not tied to one model family: latent attention with a sink, gated linear
recurrence (HGRN2), gated MLP, mixture of experts.

They take their sizes and constants as arguments and work on token rows ``[batch * positions, width]``. A mixer or
feed-forward can carry ``side`` projections: further linear maps of the same input (a block's residual gate, say) that
ride in its packed input GEMM and are handed back with the result.

``oslo_fused = False`` runs the PyTorch statements of ``ops.reference``; ``model.fuse()`` switches to the sm_100a kernels.
"""
from __future__ import annotations

from typing import Dict, NamedTuple, Optional

import torch
import torch.nn as nn
from torch import Tensor

from .. import ops
from ..parallel.layers import Linear, PackedLinear, RMSNorm
from .common import StaticKVCache


class MixerOutput(NamedTuple):
    y: Tensor                              # [rows, width]
    side: Dict[str, Tensor]                # side projections of the input
    latent: Optional[Tensor] = None        # latents other layers may read, [batch, positions, rank]
    probs: Optional[Tensor] = None         # attention weights, when asked for


class FeedForwardOutput(NamedTuple):
    y: Tensor                              # [rows, width], or one row per (token, choice)
    side: Dict[str, Tensor]
    slots: Optional[Tensor] = None         # where a (token, choice)'s row of ``y`` is; None: in order
    weights: Optional[Tensor] = None       # [rows, top] weights of those rows; None: ``y`` has one row per token


def _inference(*ts: Tensor) -> bool:
    return not (torch.is_grad_enabled() and any(t.requires_grad for t in ts))


class LatentAttention(nn.Module):
    """Attention over low-rank latents, without positions.

    ``c = norm(W_dkv h)`` (``kv_rank``) is all that is cached; per head ``k = W_uk c`` (``dim``), ``v = W_uv c`` (``vdim``),
    ``q = W_uq norm(W_dq h)`` (through ``q_rank``), scores ``(q . k) * scale``, causal. The softmax denominator also
    holds ``exp(sink[head])``; head ``h``'s output is multiplied by ``sigmoid(W_g h)[head]`` before ``W_o``. With
    ``shared_latents`` the module has no ``W_dkv`` and reads the latents of another layer (``kv_layer``).
    """

    oslo_fused = False

    def __init__(self, width: int, heads: int, dim: int, vdim: int, q_rank: int, kv_rank: int, scale: float, eps: float,
                 shared_latents: bool = False, side: Optional[Dict[str, int]] = None) -> None:
        super().__init__()
        self.heads, self.dim, self.vdim, self.kv_rank, self.scale = heads, dim, vdim, kv_rank, float(scale)
        self.shared_latents = shared_latents
        self.side = dict(side or {})
        parts = {"dq": q_rank, "g": heads, **self.side}
        if not shared_latents:
            parts["dkv"] = kv_rank
        self.in_proj = PackedLinear(width, parts)
        self.q_norm = RMSNorm(q_rank, eps)
        self.kv_norm = None if shared_latents else RMSNorm(kv_rank, eps)
        self.uq = Linear(q_rank, heads * dim, bias=False)
        self.kv_up = PackedLinear(kv_rank, {"k": heads * dim, "v": heads * vdim})
        self.sink = nn.Parameter(torch.zeros(heads))
        self.out_proj = Linear(heads * vdim, width, bias=False)

    def forward(self, h: Tensor, batch: int, layer_id: int, kv_layer: int, cache: Optional[StaticKVCache],
                latent: Optional[Tensor], keep: Optional[Tensor], output_attentions: bool = False) -> MixerOutput:
        """``h`` ``[batch * S, width]``; ``latent``: the latents of ``kv_layer`` when there is no cache; ``keep``
        ``[batch, past + S]`` marks real tokens (0 = padding)."""
        from ..ops.cuda_ops import LATENT_MAX_RANK
        p = self.in_proj(h)
        side = {n: p[n] for n in self.side}
        s = h.size(0) // batch
        if (cache is not None and s == 1 and not output_attentions and self.oslo_fused and _inference(h, self.sink)
                and ops.use_kernels(h) and self.kv_rank <= LATENT_MAX_RANK):
            return MixerOutput(self._decode(p, batch, kv_layer, cache, keep), side)
        q = self.uq(self.q_norm(p["dq"])).view(batch, s, self.heads, self.dim)
        if not self.shared_latents:
            latent = self.kv_norm(p["dkv"]).view(batch, s, self.kv_rank)
            if cache is not None:
                latent = cache.append_latent(layer_id, latent)
        elif cache is not None:
            latent = cache.latent[kv_layer][:, :cache.length + s]
        t = latent.size(1)
        kv = self.kv_up(latent.reshape(batch * t, self.kv_rank))
        k = kv["k"].view(batch, t, self.heads, self.dim)
        v = kv["v"].view(batch, t, self.heads, self.vdim)
        probs = None
        if output_attentions or not self.oslo_fused:
            o, probs = ops.reference.sink_attention(q, k, v, keep, self.sink, p["g"], self.scale)
        else:
            o = ops.sink_attention(q, k, v, keep, self.sink, p["g"], self.scale)
        return MixerOutput(self.out_proj(o), side, latent, probs if output_attentions else None)

    def _decode(self, p: Dict[str, Tensor], batch: int, kv_layer: int, cache: StaticKVCache, keep: Optional[Tensor]) -> Tensor:
        """One token per row: norms + cache append, query projection, attention over the latents, output projection."""
        from ..ops import cuda_ops
        dq = p["dq"]
        store = cache.latent_storage(kv_layer, batch, self.kv_rank, dq.dtype, dq.device, 1)
        own = not self.shared_latents
        cq = cuda_ops.latent_prep(dq, self.q_norm.weight, p["dkv"] if own else None, self.kv_norm.weight if own else None,
                                  store if own else None, cache.lengths_dev, self.q_norm.eps)
        o = cuda_ops.latent_decode(self.uq(cq), self.kv_up.part("k"), self.kv_up.part("v"), store, cache.lengths_next, keep,
                                   self.sink, p["g"], self.scale, self.heads)
        return self.out_proj(o)


class GatedLinearRecurrence(nn.Module):
    """HGRN2: linear attention with a data-dependent forget gate that also decides what is written.

    Per head ``q = silu(W_q h)`` (``dim``), ``v = W_v h`` (``vdim``), ``f = lower + (1 - lower) sigmoid(W_f h + b_f)``;
    ``S <- diag(f) S + (1 - f) v^T``, ``o = S^T q``; ``o`` is RMS-normed per head and projected. ``S`` is fp32.
    """

    oslo_fused = False

    def __init__(self, width: int, heads: int, dim: int, vdim: int, eps: float, side: Optional[Dict[str, int]] = None) -> None:
        super().__init__()
        self.heads, self.dim, self.vdim = heads, dim, vdim
        self.side = dict(side or {})
        self.in_proj = PackedLinear(width, {"q": heads * dim, "f": heads * dim, "v": heads * vdim, **self.side})
        self.f_bias = nn.Parameter(torch.zeros(heads * dim))
        self.lower = nn.Parameter(torch.zeros(heads * dim))
        self.o_norm = RMSNorm(vdim, eps)
        self.out_proj = Linear(heads * vdim, width, bias=False)

    def forward(self, h: Tensor, batch: int, layer_id: int, cache: Optional[StaticKVCache], keep: Optional[Tensor]) -> MixerOutput:
        p = self.in_proj(h)
        s = h.size(0) // batch
        state = None
        if cache is not None:
            state = cache.recurrent_state(layer_id, (batch, self.heads, self.dim, self.vdim), h.device)
        if keep is not None:
            keep = keep[:, -s:]
        fn = ops.gated_recurrence if self.oslo_fused else _plain_recurrence
        o = fn(p["q"], p["f"], p["v"], self.f_bias, self.lower, self.o_norm.weight, self.o_norm.eps, batch, self.heads, keep, state)
        return MixerOutput(self.out_proj(o), {n: p[n] for n in self.side})


def _plain_recurrence(q, f, v, f_bias, lower, norm_w, eps, batch, heads, keep, state):
    dim, vdim = q.size(-1) // heads, v.size(-1) // heads
    o, final = ops.reference.recurrence(q, f, v, f_bias, lower, keep, state, batch, heads, dim, vdim)
    if state is not None:
        state.copy_(final.detach())
    return ops.reference.rms_norm(o, norm_w, eps).reshape(-1, heads * vdim)


class GatedMLP(nn.Module):
    """``W_down (silu(W_gate h) * (W_up h))``."""

    oslo_fused = False

    def __init__(self, width: int, ff: int, side: Optional[Dict[str, int]] = None) -> None:
        super().__init__()
        self.side = dict(side or {})
        self.in_proj = PackedLinear(width, {"gate": ff, "up": ff, **self.side})
        self.down = Linear(ff, width, bias=False)

    def forward(self, h: Tensor) -> FeedForwardOutput:
        p = self.in_proj(h)
        a = (ops.silu_mul if self.oslo_fused else ops.reference.silu_mul)(p["gate"], p["up"])
        return FeedForwardOutput(self.down(a), {n: p[n] for n in self.side})


class MixtureOfExperts(nn.Module):
    """``experts`` small feed-forwards ``W_down relu(W_up h)^2``; a token's router logits ``W_r h + b`` (fp32) choose ``top`` of
    them, weighted by the softmax over the chosen logits only. No capacity limit: every choice is computed. The result keeps
    one row per (token, choice); whoever adds it to the residual stream sums the rows."""

    oslo_fused = False

    def __init__(self, width: int, ff: int, experts: int, top: int, side: Optional[Dict[str, int]] = None) -> None:
        super().__init__()
        self.experts, self.top = experts, top
        self.side = dict(side or {})
        self.in_proj = PackedLinear(width, self.side) if self.side else None
        self.router = Linear(width, experts)
        self.up = nn.Parameter(torch.empty(experts, ff, width).normal_(std=0.02))
        self.down = nn.Parameter(torch.empty(experts, width, ff).normal_(std=0.02))

    def forward(self, h: Tensor) -> FeedForwardOutput:
        side = self.in_proj(h) if self.in_proj is not None else {}
        if self.oslo_fused:
            idx, weights = ops.moe_route(h, self.router.weight, self.router.bias, self.top)
            y, slots = ops.moe_experts(h, idx, self.up, self.down)
        else:
            idx, weights = ops.reference.moe_route(h, self.router.weight, self.router.bias, self.top)
            y, slots = ops.reference.moe_experts(h, idx, self.up, self.down), None
        return FeedForwardOutput(y, side, slots, weights)
