"""Token mixers and feed-forwards that are not tied to one model family: latent attention with a sink, grouped-query attention
with query / key norms and capped scores, gated linear recurrence (HGRN2), linear attention with constant decays, linear
recurrence with a bonus (WKV), selective scan (Mamba), two mixers side by side; gated MLPs, mixture of experts.

They take their sizes and constants as arguments and work on token rows ``[batch * positions, width]``. A mixer or
feed-forward can carry ``side`` projections: further linear maps of the same input (a block's residual gate, say) that
ride in its packed input GEMM and are handed back with the result.

``oslo_fused = False`` runs the PyTorch statements of ``ops.reference``; ``model.fuse()`` switches to the sm_100a kernels.
"""
from __future__ import annotations

import math
from typing import Any, Dict, NamedTuple, Optional, Sequence, Tuple

import torch
import torch.nn as nn
from torch import Tensor

from .. import ops
from ..parallel.layers import Linear, PackedLinear, RMSNorm, StackedLinear
from .common import StaticKVCache


class Branch(NamedTuple):
    """A result on its way to the residual stream: ``factor * y``, or ``factor * norm(y) * norm_weight``."""
    y: Tensor                              # [rows, width]
    norm_weight: Optional[Tensor] = None
    factor: float = 1.0


class MixerOutput(NamedTuple):
    y: Optional[Tensor]                    # [rows, width]; None: the result is the sum of ``branches``
    side: Dict[str, Tensor]                # side projections of the input
    latent: Optional[Tensor] = None        # latents other layers may read, [batch, positions, rank]
    probs: Optional[Tensor] = None         # attention weights, when asked for
    branches: Tuple[Branch, ...] = ()


class FeedForwardOutput(NamedTuple):
    y: Tensor                              # [rows, width], or one row per (token, choice)
    side: Dict[str, Tensor]
    slots: Optional[Tensor] = None         # where a (token, choice)'s row of ``y`` is; None: in order
    weights: Optional[Tensor] = None       # [rows, top] weights of those rows; None: ``y`` has one row per token


def _inference(*ts: Tensor) -> bool:
    return not (torch.is_grad_enabled() and any(t.requires_grad for t in ts))


def _last(keep: Optional[Tensor], s: int) -> Optional[Tensor]:
    """The columns of ``keep`` ``[batch, past + s]`` that belong to this call."""
    return None if keep is None else keep[:, -s:]


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
        keep = _last(keep, s)
        fn = ops.gated_recurrence if self.oslo_fused else _plain_recurrence
        o = fn(p["q"], p["f"], p["v"], self.f_bias, self.lower, self.o_norm.weight, self.o_norm.eps, batch, self.heads, keep, state)
        return MixerOutput(self.out_proj(o), {n: p[n] for n in self.side})


def _plain_recurrence(q, f, v, f_bias, lower, norm_w, eps, batch, heads, keep, state):
    dim, vdim = q.size(-1) // heads, v.size(-1) // heads
    o, final = ops.reference.recurrence(q, f, v, f_bias, lower, keep, state, batch, heads, dim, vdim)
    if state is not None:
        state.copy_(final.detach())
    return ops.reference.rms_norm(o, norm_w, eps).reshape(-1, heads * vdim)


class _Constants:
    """Vectors that the configuration fixes, as fp32 tensors on whatever device they are asked for (not parameters: neither
    saved nor converted to the model's storage type)."""

    def _constant(self, name: str, values: Sequence[float], device) -> Tensor:
        table = self.__dict__.setdefault("_constant_tensors", {})
        key = (name, str(device))
        if key not in table:
            table[key] = torch.tensor(list(values), dtype=torch.float32, device=device)
        return table[key]


class GroupedQueryAttention(nn.Module, _Constants):
    """Causal softmax attention with ``heads`` query heads over ``kv_heads`` key / value heads.

    Queries and keys are RMS-normed per head (weights ``[dim]``, shared by the heads), then the first ``rot_dims`` dims are rotated
    (interleaved pairs, ``rot_base``); scores ``(q . k) * scale`` pass through ``softcap * tanh(score / softcap)`` (0: they do
    not); the softmax denominator holds an additional 1 (a sink with score 0). Keys (after norm and rotation) and values are
    cached. ``in_proj=False``: the projections come from the caller's packed GEMM (``parts``)."""

    oslo_fused = False

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, eps: float, rot_dims: int = 0,
                 rot_base: float = 10000.0, softcap: float = 0.0, in_proj: bool = True) -> None:
        super().__init__()
        if heads % kv_heads:
            raise ValueError(f"{heads} query heads do not divide into {kv_heads} groups")
        self.heads, self.kv_heads, self.dim, self.vdim = heads, kv_heads, dim, vdim
        self.scale, self.softcap = float(scale), float(softcap)
        self.frequencies = ops.reference.rotary_frequencies(rot_dims, rot_base)
        self.parts = {"q": heads * dim, "k": kv_heads * dim, "v": kv_heads * vdim}
        self.in_proj = PackedLinear(width, self.parts) if in_proj else None
        self.q_norm = RMSNorm(dim, eps)
        self.k_norm = RMSNorm(dim, eps)
        self.out_proj = Linear(heads * vdim, width, bias=False)

    def forward(self, h: Tensor, batch: int, layer_id: int, cache: Optional[StaticKVCache], keep: Optional[Tensor],
                positions: Tensor, output_attentions: bool = False) -> MixerOutput:
        return self.mix(self.in_proj(h), batch, layer_id, cache, keep, positions, output_attentions)

    def mix(self, p: Dict[str, Tensor], batch: int, layer_id: int, cache: Optional[StaticKVCache], keep: Optional[Tensor],
            positions: Tensor, output_attentions: bool = False) -> MixerOutput:
        """``keep`` ``[batch, past + S]`` marks real tokens, ``positions`` ``[batch, S]``."""
        rows = p["q"].size(0)
        s = rows // batch
        freq = self._constant("freq", self.frequencies, p["q"].device)
        sink = self._sink(p["q"])
        if (self.oslo_fused and not output_attentions and _inference(p["q"], self.q_norm.weight) and ops.use_kernels(p["q"])):
            o = self._kernels(p, batch, s, layer_id, cache, keep, positions, freq, sink)
            return MixerOutput(self.out_proj(o), {})
        q = ops.reference.norm_rotate(p["q"].reshape(batch, s, self.heads, self.dim), self.q_norm.weight, self.q_norm.eps, positions, freq)
        k = ops.reference.norm_rotate(p["k"].reshape(batch, s, self.kv_heads, self.dim), self.k_norm.weight, self.k_norm.eps, positions, freq)
        v = p["v"].reshape(batch, s, self.kv_heads, self.vdim)
        if cache is not None:
            k, v, end = cache.append(layer_id, k.transpose(1, 2), v.transpose(1, 2))
            if s == 1 and not output_attentions:
                o = ops.reference.grouped_decode(q[:, 0], k, v, cache.lengths_next, keep, sink, self.scale, self.softcap)
                return MixerOutput(self.out_proj(o), {})
            k, v = k[:, :, :end].transpose(1, 2), v[:, :, :end].transpose(1, 2)
        o, probs = ops.reference.sink_attention(q, k, v, keep, sink, None, self.scale, self.softcap)
        return MixerOutput(self.out_proj(o), {}, probs=probs if output_attentions else None)

    def _sink(self, like: Tensor) -> Tensor:
        table = self.__dict__.setdefault("_constant_tensors", {})
        key = ("sink", str(like.device), like.dtype)
        if key not in table:
            table[key] = torch.zeros(self.heads, dtype=like.dtype, device=like.device)
        return table[key]

    def _kernels(self, p, batch, s, layer_id, cache, keep, positions, freq, sink) -> Tensor:
        """Norms, rotation and cache append in one launch, then the prompt or the decode kernel on the cached keys."""
        from ..ops import cuda_ops
        q = p["q"]
        holder = cache if cache is not None else StaticKVCache(s)
        ks, vs = holder.kv_storage(layer_id, batch, self.kv_heads, self.dim, self.vdim, q.dtype, q.device, s)
        q = cuda_ops.qkv_prep(q, p["k"], p["v"], self.q_norm.weight, self.k_norm.weight, self.q_norm.eps, positions, freq, ks, vs,
                              holder.lengths_dev)
        if s == 1 and cache is not None:
            return cuda_ops.grouped_decode(q[:, 0], ks, vs, holder.lengths_next, keep, sink, self.scale, self.softcap)
        end = holder.length + s
        return cuda_ops.sink_attention(q, ks[:, :, :end].transpose(1, 2), vs[:, :, :end].transpose(1, 2), keep, sink, None, self.scale,
                                       self.softcap)


class DecayedLinearAttention(nn.Module, _Constants):
    """Linear attention with one constant decay per head (Lightning attention): ``q``, ``k``, ``v`` are ``silu`` of their projections,
    ``S <- decay S + k v^T`` (fp32), ``o = S^T q``; the heads together are RMS-normed, multiplied by ``sigmoid(W_g h)`` and
    projected. ``in_proj=False``: the projections come from the caller's packed GEMM (``parts``)."""

    oslo_fused = False

    def __init__(self, width: int, heads: int, dim: int, vdim: int, decay: Sequence[float], eps: float, in_proj: bool = True) -> None:
        super().__init__()
        if len(decay) != heads:
            raise ValueError(f"{len(decay)} decays for {heads} heads")
        self.heads, self.dim, self.vdim = heads, dim, vdim
        self.decay = [float(d) for d in decay]
        self.parts = {"q": heads * dim, "k": heads * dim, "v": heads * vdim, "g": heads * vdim}
        self.in_proj = PackedLinear(width, self.parts) if in_proj else None
        self.o_norm = RMSNorm(heads * vdim, eps)
        self.out_proj = Linear(heads * vdim, width, bias=False)

    def forward(self, h: Tensor, batch: int, layer_id: int, cache: Optional[StaticKVCache], keep: Optional[Tensor]) -> MixerOutput:
        return self.mix(self.in_proj(h), batch, layer_id, cache, keep)

    def mix(self, p: Dict[str, Tensor], batch: int, layer_id: int, cache: Optional[StaticKVCache], keep: Optional[Tensor]) -> MixerOutput:
        s = p["q"].size(0) // batch
        state = None
        if cache is not None:
            state = cache.recurrent_state(layer_id, (batch, self.heads, self.dim, self.vdim), p["q"].device)
        o = ops.decayed_attention(p["q"], p["k"], p["v"], self._constant("decay", self.decay, p["q"].device), _last(keep, s), state,
                                  batch, self.heads, fused=self.oslo_fused)
        o = ops.gated_rms_norm(o, self.o_norm.weight, p["g"], self.o_norm.eps, self.heads * self.vdim, "sigmoid", fused=self.oslo_fused)
        return MixerOutput(self.out_proj(o), {})


class SideBySide(nn.Module):
    """Grouped-query attention and linear attention with constant decays on the same input, from one packed GEMM; the result is
    half the sum of the two, each RMS-normed over the model width first (left to whoever adds it to the residual stream)."""

    def __init__(self, width: int, left: Dict[str, Any], right: Dict[str, Any], eps: float) -> None:
        super().__init__()
        self.left = GroupedQueryAttention(width, eps=eps, in_proj=False, **left)
        self.right = DecayedLinearAttention(width, eps=eps, in_proj=False, **right)
        self.in_proj = PackedLinear(width, {f"{side}.{n}": size for side in ("left", "right")
                                            for n, size in getattr(self, side).parts.items()})
        self.left_norm = RMSNorm(width, eps)
        self.right_norm = RMSNorm(width, eps)

    def forward(self, h: Tensor, batch: int, layer_id: int, cache: Optional[StaticKVCache], keep: Optional[Tensor],
                positions: Tensor, output_attentions: bool = False) -> MixerOutput:
        p = self.in_proj(h)
        of = lambda side: {n: p[f"{side}.{n}"] for n in getattr(self, side).parts}              # noqa: E731
        left = self.left.mix(of("left"), batch, layer_id, cache, keep, positions, output_attentions)
        right = self.right.mix(of("right"), batch, layer_id, cache, keep)
        return MixerOutput(None, {}, probs=left.probs, branches=(Branch(left.y, self.left_norm.weight, 0.5),
                                                                 Branch(right.y, self.right_norm.weight, 0.5)))


class BonusRecurrence(nn.Module):
    """RWKV-style time mixing: every projection reads its own mix ``h + (h' - h) mu`` of the token and the one before it; per head
    ``o = (S + diag(u) k v^T)^T r``, then ``S <- diag(w) S + k v^T`` (fp32) with ``w = exp(-exp(W_w2 tanh(W_w1 mix) + w0))``; heads are
    divided by their root mean square, times a weight, times ``silu`` of the gate projection, and projected."""

    oslo_fused = False
    MIXES = ("r", "k", "v", "g", "w")

    def __init__(self, width: int, heads: int, dim: int, eps: float, decay_rank: int = 64) -> None:
        super().__init__()
        self.heads, self.dim, self.eps = heads, dim, float(eps)
        n = heads * dim
        self.mu = nn.Parameter(torch.full((len(self.MIXES), width), 0.5))
        self.rkvg = StackedLinear(4, width, n)
        self.w1 = Linear(width, decay_rank, bias=False)
        self.w2 = Linear(decay_rank, n, bias=False)
        self.w0 = nn.Parameter(torch.linspace(-6.0, -1.0, n))
        self.u = nn.Parameter(torch.zeros(n))
        self.o_norm = nn.Parameter(torch.ones(n))
        self.out_proj = Linear(n, width, bias=False)

    def set_decay_rank(self, rank: int) -> None:
        """Another rank for the decay's projection pair (checkpoints may fix it by their shapes alone)."""
        if rank != self.w1.out_features:
            like = self.w1.weight
            self.w1 = Linear(self.w1.in_features, rank, bias=False, device=like.device, dtype=like.dtype)
            self.w2 = Linear(rank, self.w2.out_features, bias=False, device=like.device, dtype=like.dtype)

    def forward(self, h: Tensor, batch: int, layer_id: int, cache: Optional[StaticKVCache], keep: Optional[Tensor]) -> MixerOutput:
        s = h.size(0) // batch
        keep = _last(keep, s)
        prev = state = None
        if cache is not None:
            prev = cache.recurrent_state(layer_id, (batch, h.size(1)), h.device, "shift")
            state = cache.recurrent_state(layer_id, (batch, self.heads, self.dim, self.dim), h.device)
        mixed = ops.token_shift(h, self.mu, batch, keep, prev, fused=self.oslo_fused)
        r, k, v, g = self.rkvg(mixed[:4])
        t = self.w1(mixed[4])
        if s == 1 and state is not None and self.oslo_fused and _inference(h, self.w0) and ops.use_kernels(h):
            from ..ops import cuda_ops
            o = cuda_ops.bonus_step(r, k, v, t, self.w2.weight, self.w0, self.u, self.o_norm, g, keep, state, self.eps, self.heads)
            return MixerOutput(self.out_proj(o), {})
        z = ops.linear_fp32(torch.tanh(t.to(torch.float32)).to(t.dtype), self.w2.weight, fused=self.oslo_fused)
        o = ops.bonus_recurrence(r, k, v, z, self.w0, self.u, keep, state, batch, self.heads, fused=self.oslo_fused)
        o = ops.gated_rms_norm(o, self.o_norm, g, self.eps, self.dim, "silu", fused=self.oslo_fused)
        return MixerOutput(self.out_proj(o), {})


class SelectiveScan(nn.Module):
    """Mamba: ``x`` and ``z`` from one projection; ``x`` through a causal convolution per channel and ``silu``; steps ``dt`` and the
    token's ``B``, ``C`` from ``x``; ``S <- exp(dt A) S + dt x B`` per channel and state (fp32), ``y = S C + D x``, times ``silu(z)``."""

    oslo_fused = False

    def __init__(self, width: int, inner: int, state: int, dt_rank: int, conv: int) -> None:
        super().__init__()
        self.inner, self.state, self.dt_rank, self.taps = inner, state, dt_rank, conv
        self.in_proj = PackedLinear(width, {"x": inner, "z": inner})
        self.conv_weight = nn.Parameter(torch.empty(inner, conv).normal_(std=conv ** -0.5))
        self.conv_bias = nn.Parameter(torch.zeros(inner))
        self.x_proj = PackedLinear(inner, {"dt": dt_rank, "b": state, "c": state})
        self.dt_proj = Linear(dt_rank, inner, bias=False)
        self.dt_bias = nn.Parameter(torch.linspace(math.log(math.expm1(1e-3)), math.log(math.expm1(0.1)), inner))
        self.a_log = nn.Parameter(torch.log(torch.arange(1.0, state + 1.0)).repeat(inner, 1))
        self.d = nn.Parameter(torch.ones(inner))
        self.out_proj = Linear(inner, width, bias=False)

    def forward(self, h: Tensor, batch: int, layer_id: int, cache: Optional[StaticKVCache], keep: Optional[Tensor]) -> MixerOutput:
        s = h.size(0) // batch
        keep = _last(keep, s)
        prev = state = None
        if cache is not None:
            prev = cache.recurrent_state(layer_id, (batch, self.taps - 1, self.inner), h.device, "conv")
            state = cache.recurrent_state(layer_id, (batch, self.inner, self.state), h.device)
        p = self.in_proj(h)
        x = ops.causal_conv_silu(p["x"], self.conv_weight, self.conv_bias, batch, keep, prev, fused=self.oslo_fused)
        sel = self.x_proj(x)
        if s == 1 and state is not None and self.oslo_fused and _inference(h, self.a_log) and ops.use_kernels(h):
            from ..ops import cuda_ops
            y = cuda_ops.scan_step(x, sel["dt"], self.dt_proj.weight, self.dt_bias, self.a_log, sel["b"], sel["c"], self.d, p["z"], keep,
                                   state)
            return MixerOutput(self.out_proj(y), {})
        dt = ops.linear_fp32(sel["dt"], self.dt_proj.weight, fused=self.oslo_fused)
        y = ops.selective_scan(x, dt, self.dt_bias, self.a_log, sel["b"], sel["c"], self.d, p["z"], batch, keep, state,
                               fused=self.oslo_fused)
        return MixerOutput(self.out_proj(y), {})


class GatedMLP(nn.Module):
    """``W_down act(W_gate h, W_up h)``: ``silu(gate) * up``, or with a ``limit`` the clamped unit ``g sigmoid(alpha g) (u + 1)``
    of ``g = min(gate, limit)``, ``u = clamp(up, -limit, limit)``."""

    oslo_fused = False

    def __init__(self, width: int, ff: int, side: Optional[Dict[str, int]] = None, limit: Optional[float] = None,
                 alpha: float = 1.702) -> None:
        super().__init__()
        self.limit, self.alpha = (None if limit is None else float(limit)), float(alpha)
        self.side = dict(side or {})
        self.in_proj = PackedLinear(width, {"gate": ff, "up": ff, **self.side})
        self.down = Linear(ff, width, bias=False)

    def forward(self, h: Tensor) -> FeedForwardOutput:
        p = self.in_proj(h)
        if self.limit is not None:
            a = ops.clamped_glu(p["gate"], p["up"], self.limit, self.alpha, fused=self.oslo_fused)
        else:
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
