"""Token mixers and feed-forwards that are not tied to one model family: latent attention (with or without a sink and a rotated
part), grouped-query attention with query / key norms, capped or mixed scores, windows and gates, gated linear recurrence (HGRN2),
linear attention with constant decays, linear recurrence with a bonus (WKV), matrix memory (mLSTM), selective scan (Mamba), two
mixers side by side; dense and gated MLPs, mixtures of experts; causal convolutions of a mixer's input, per-token inputs of a layer; residual
streams with hyper-connections.

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
from ..ops.reference import Branch
from ..parallel.layers import Linear, PackedLinear, RMSNorm, StackedLinear
from .common import StaticKVCache


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
    choice: Optional[Tensor] = None        # [rows, top] chosen router outputs, when some of them are no experts
    shared: Optional[Tensor] = None        # [rows, width] of a shared expert, to be added times sigmoid(shared_gate)
    shared_gate: Optional[Tensor] = None   # [rows, 1]


def _inference(*ts: Tensor) -> bool:
    return not (torch.is_grad_enabled() and any(t.requires_grad for t in ts))


def _last(keep: Optional[Tensor], s: int) -> Optional[Tensor]:
    """The columns of ``keep`` ``[batch, past + s]`` that belong to this call."""
    return None if keep is None else keep[:, -s:]


class _Constants:
    """Vectors that the configuration fixes, as fp32 tensors on whatever device they are asked for (not parameters: neither
    saved nor converted to the model's storage type)."""

    def _constant(self, name: str, values: Sequence[float], device) -> Tensor:
        table = self.__dict__.setdefault("_constant_tensors", {})
        key = (name, str(device))
        if key not in table:
            table[key] = torch.tensor(list(values), dtype=torch.float32, device=device)
        return table[key]


class LatentAttention(nn.Module, _Constants):
    """Attention over low-rank latents.

    ``c = norm(W_dkv h)`` (``kv_rank``) is what is cached; per head ``k = W_uk c`` (``dim``), ``v = W_uv c`` (``vdim``), ``q = W_uq
    norm(W_dq h)`` (through ``q_rank``), scores ``(q . k) * scale``, causal. With ``rot_dim`` a head's query has ``rot_dim`` further
    dimensions and ``W_dkv h`` as many further rows, one key part for all heads (not normed, cached with ``c``); both are rotated
    (halves, ``rot_base``) and their product joins the score. With ``sink`` the softmax denominator also holds ``exp(sink[head])``. The
    output is multiplied by ``sigmoid(W_g h)`` before ``W_o``: one number per head, or (``gate="element"``) one per element. With
    ``shared_latents`` the module has no ``W_dkv`` and reads the latents of another layer (``kv_layer``).
    """

    oslo_fused = False

    def __init__(self, width: int, heads: int, dim: int, vdim: int, q_rank: int, kv_rank: int, scale: float, eps: float,
                 shared_latents: bool = False, side: Optional[Dict[str, int]] = None, rot_dim: int = 0, rot_base: float = 10000.0,
                 sink: bool = True, gate: str = "head") -> None:
        super().__init__()
        if gate not in ("head", "element"):
            raise ValueError(f"output gate per {gate!r}")
        self.heads, self.dim, self.vdim, self.kv_rank, self.scale = heads, dim, vdim, kv_rank, float(scale)
        self.rot_dim = rot_dim
        self.frequencies = ops.reference.rotary_frequencies(rot_dim, rot_base)
        self.shared_latents = shared_latents
        self.side = dict(side or {})
        parts = {"dq": q_rank, "g": heads if gate == "head" else heads * vdim, **self.side}
        if not shared_latents:
            parts["dkv"] = kv_rank + rot_dim
        self.in_proj = PackedLinear(width, parts)
        self.q_norm = RMSNorm(q_rank, eps)
        self.kv_norm = None if shared_latents else RMSNorm(kv_rank, eps)
        self.uq = Linear(q_rank, heads * (dim + rot_dim), bias=False)
        self.kv_up = PackedLinear(kv_rank, {"k": heads * dim, "v": heads * vdim})
        self.sink = nn.Parameter(torch.zeros(heads)) if sink else None
        self.out_proj = Linear(heads * vdim, width, bias=False)

    def forward(self, h: Tensor, batch: int, layer_id: int, kv_layer: int, cache: Optional[StaticKVCache],
                latent: Optional[Tensor], keep: Optional[Tensor], output_attentions: bool = False,
                positions: Optional[Tensor] = None) -> MixerOutput:
        """``h`` ``[batch * S, width]``; ``latent``: the latents of ``kv_layer`` when there is no cache; ``keep``
        ``[batch, past + S]`` marks real tokens (0 = padding); ``positions`` ``[batch, S]`` where something is rotated."""
        from ..ops.cuda_ops import LATENT_MAX_RANK
        p = self.in_proj(h)
        side = {n: p[n] for n in self.side}
        s = h.size(0) // batch
        kernels = self.oslo_fused and not output_attentions and _inference(h, self.out_proj.weight) and ops.use_kernels(h)
        if cache is not None and s == 1 and kernels and self.kv_rank <= LATENT_MAX_RANK:
            return MixerOutput(self._decode(p, batch, kv_layer, cache, keep, positions), side)
        if self.rot_dim and kernels and not self.shared_latents:
            q, latent, c = self._prompt(p, batch, s, layer_id, cache, positions)
        else:
            q = self.uq(self.q_norm(p["dq"])).view(batch, s, self.heads, self.dim + self.rot_dim)
            if self.rot_dim:
                freq = self._constant("freq", self.frequencies, h.device)
                turned = ops.reference.rotate_halves(q[..., self.dim:], positions, freq)
                q = torch.cat([q[..., :self.dim], turned], dim=-1)
            if not self.shared_latents:
                latent = self.kv_norm(p["dkv"][:, :self.kv_rank]).view(batch, s, self.kv_rank)
                if self.rot_dim:
                    shared = p["dkv"][:, self.kv_rank:].reshape(batch, s, 1, self.rot_dim)
                    latent = torch.cat([latent, ops.reference.rotate_halves(shared, positions, freq)[:, :, 0]], dim=-1)
                if cache is not None:
                    latent = cache.append_latent(layer_id, latent)
            elif cache is not None:
                latent = cache.latent[kv_layer][:, :cache.length + s]
            c = latent[..., :self.kv_rank].reshape(-1, self.kv_rank)
        t = latent.size(1)
        kv = self.kv_up(c)
        k = kv["k"].view(batch, t, self.heads, self.dim)
        v = kv["v"].view(batch, t, self.heads, self.vdim)
        rotated = (q[..., self.dim:], latent[..., self.kv_rank:]) if self.rot_dim else (None, None)
        args = (q[..., :self.dim], k, v, keep, self.sink, p["g"], self.scale, 0.0, 0, 0, None, *rotated)
        probs = None
        if output_attentions or not self.oslo_fused:
            o, probs = ops.reference.sink_attention(*args)
        else:
            o = ops.sink_attention(*args)
        return MixerOutput(self.out_proj(o), side, latent, probs if output_attentions else None)

    def _prompt(self, p: Dict[str, Tensor], batch: int, s: int, layer_id: int, cache: Optional[StaticKVCache], positions: Tensor):
        """Norms, rotations and cache append of a prompt: queries ``[batch, S, heads, *]``, what the cache holds now, and the latents of
        that as contiguous rows."""
        from ..ops import cuda_ops
        dq = p["dq"]
        freq = self._constant("freq", self.frequencies, dq.device)
        holder = cache if cache is not None else StaticKVCache(s)
        store = holder.latent_storage(layer_id, batch, self.kv_rank + self.rot_dim, dq.dtype, dq.device, s)
        cq, c = cuda_ops.latent_prep(dq, self.q_norm.weight, p["dkv"], self.kv_norm.weight, store, holder.lengths_dev, self.q_norm.eps,
                                     positions, freq, rows=True)
        q = cuda_ops.rotate_halves_(self.uq(cq).view(batch, s, self.heads, self.dim + self.rot_dim), positions, freq)
        latent = store[:, :holder.length + s]
        if holder.length:
            c = latent[..., :self.kv_rank].reshape(-1, self.kv_rank)
        return q, latent, c

    def _decode(self, p: Dict[str, Tensor], batch: int, kv_layer: int, cache: StaticKVCache, keep: Optional[Tensor],
                positions: Optional[Tensor]) -> Tensor:
        """One token per row: norms + rotation + cache append, query projection, attention over the latents, output projection."""
        from ..ops import cuda_ops
        dq = p["dq"]
        store = cache.latent_storage(kv_layer, batch, self.kv_rank + self.rot_dim, dq.dtype, dq.device, 1)
        own = not self.shared_latents
        freq = self._constant("freq", self.frequencies, dq.device) if self.rot_dim else None
        cq, _ = cuda_ops.latent_prep(dq, self.q_norm.weight, p["dkv"] if own else None, self.kv_norm.weight if own else None,
                                     store if own else None, cache.lengths_dev, self.q_norm.eps, positions, freq)
        o = cuda_ops.latent_decode(self.uq(cq), self.kv_up.part("k"), self.kv_up.part("v"), store, cache.lengths_next, keep,
                                   self.sink, p["g"], self.scale, self.heads, positions, freq)
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


class GroupedQueryAttention(nn.Module, _Constants):
    """Causal softmax attention with ``heads`` query heads over ``kv_heads`` key / value heads.

    Queries and keys are RMS-normed per head (weights ``[dim]``, shared by the heads; ``norm_weights=False``: without weights), then
    the first ``rot_dims`` dims are rotated (interleaved pairs, or ``halves``: dim ``i`` with dim ``i + rot_dims / 2``; ``rot_base``, YaRN
    ``rot_scaling``); scores ``(q . k) * scale`` pass through ``softcap * tanh(score / softcap)`` (0: they do not). With ``sink`` the softmax
    denominator holds an additional 1 (a sink with score 0). With a ``window`` > 0 a position reads the last ``window`` positions and the
    first ``keep_first`` of the sequence. ``value_is_key``: values are the projected keys, before norm and rotation. ``gate``: ``"head"``
    (head ``h``'s output is multiplied by ``sigmoid(W_g x)[h]``), ``"element"`` (one factor per element) or ``None``. ``talk``: before the
    softmax the heads' scores are mixed, ``score_h <- sum_g talk[h, g] score_g``; the mix is folded into the queries
    (``reference.norm_rotate_fold``) and the keys of all key heads are cached as one row per token. Keys (after norm and rotation)
    and values are cached. ``in_proj=False``: the projections come from the caller's packed GEMM (``parts``)."""

    oslo_fused = False

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, eps: float, rot_dims: int = 0,
                 rot_base: float = 10000.0, softcap: float = 0.0, in_proj: bool = True, norm_weights: bool = True, sink: bool = True,
                 window: int = 0, keep_first: int = 0, value_is_key: bool = False, gate: Optional[str] = None, halves: bool = False,
                 rot_scaling: Optional[Dict[str, float]] = None, talk: bool = False) -> None:
        super().__init__()
        if heads % kv_heads:
            raise ValueError(f"{heads} query heads do not divide into {kv_heads} groups")
        if value_is_key and vdim != dim:
            raise ValueError(f"values are the keys, but have size {vdim} and not {dim}")
        if gate not in (None, "head", "element"):
            raise ValueError(f"output gate per {gate!r}")
        self.heads, self.kv_heads, self.dim, self.vdim, self.eps = heads, kv_heads, dim, vdim, float(eps)
        self.scale, self.softcap = float(scale), float(softcap)
        self.sink, self.window, self.keep_first = bool(sink), int(window), int(keep_first)
        self.frequencies = ops.reference.rotary_frequencies(rot_dims, rot_base, rot_scaling)
        self.halves, self.amplitude = bool(halves), ops.reference.rotary_amplitude(rot_scaling)
        self.parts = {"q": heads * dim, "k": kv_heads * dim}
        if not value_is_key:
            self.parts["v"] = kv_heads * vdim
        if gate is not None:
            self.parts["g"] = heads if gate == "head" else heads * vdim
        self.in_proj = PackedLinear(width, self.parts) if in_proj else None
        self.q_norm = RMSNorm(dim, eps) if norm_weights else None
        self.k_norm = RMSNorm(dim, eps) if norm_weights else None
        self.talk = nn.Parameter(torch.eye(heads)) if talk else None
        self.out_proj = Linear(heads * vdim, width, bias=False)

    def forward(self, h: Tensor, batch: int, layer_id: int, cache: Optional[StaticKVCache], keep: Optional[Tensor],
                positions: Tensor, output_attentions: bool = False, lead: Optional[Tensor] = None) -> MixerOutput:
        return self.mix(self.in_proj(h), batch, layer_id, cache, keep, positions, output_attentions, lead)

    def mix(self, p: Dict[str, Tensor], batch: int, layer_id: int, cache: Optional[StaticKVCache], keep: Optional[Tensor],
            positions: Tensor, output_attentions: bool = False, lead: Optional[Tensor] = None) -> MixerOutput:
        """``keep`` ``[batch, past + S]`` marks real tokens, ``positions`` ``[batch, S]``; ``lead`` ``[batch]`` int32: padding ahead of a
        sequence's first token (``None``: none anywhere)."""
        rows = p["q"].size(0)
        s = rows // batch
        freq = self._constant("freq", self.frequencies, p["q"].device)
        sink, gate, values = self._sink(p["q"]), p.get("g"), p.get("v", p["k"])
        wq, wk = (None, None) if self.q_norm is None else (self.q_norm.weight, self.k_norm.weight)
        mask = (self.window, self.keep_first, lead)
        if (self.oslo_fused and not output_attentions and _inference(p["q"], self.out_proj.weight) and ops.use_kernels(p["q"])):
            o = self._kernels(p, values, batch, s, layer_id, cache, keep, positions, freq, sink, gate, mask)
            return MixerOutput(self.out_proj(o), {})
        q, turn = p["q"].reshape(batch, s, self.heads, self.dim), (self.halves, self.amplitude)
        if self.talk is None:
            q = ops.reference.norm_rotate(q, wq, self.eps, positions, freq, *turn)
        else:
            q = ops.reference.norm_rotate_fold(q, wq, self.eps, positions, freq, self.talk, self.kv_heads, *turn)
        k = ops.reference.norm_rotate(p["k"].reshape(batch, s, self.kv_heads, self.dim), wk, self.eps, positions, freq, *turn)
        v = values.reshape(batch, s, self.kv_heads, self.vdim)
        if self.talk is not None:
            k = k.flatten(2).unsqueeze(2)
        if cache is not None:
            kc, vc = (k, v) if self.talk is None else (k, v.flatten(2).unsqueeze(2))
            k, v, end = cache.append(layer_id, kc.transpose(1, 2), vc.transpose(1, 2))
            v = v if self.talk is None else self._heads(v, self.vdim)
            if s == 1 and not output_attentions:
                o = ops.reference.grouped_decode(q[:, 0], k, v, cache.lengths_next, keep, sink, self.scale, self.softcap, gate, *mask)
                return MixerOutput(self.out_proj(o), {})
            k, v = k[:, :, :end].transpose(1, 2), v[:, :, :end].transpose(1, 2)
        o, probs = ops.reference.sink_attention(q, k, v, keep, sink, gate, self.scale, self.softcap, *mask)
        return MixerOutput(self.out_proj(o), {}, probs=probs if output_attentions else None)

    def _heads(self, store: Tensor, dim: int) -> Tensor:
        """A cache with all key heads in a row, ``[B, 1, T, kv_heads * dim]``, as ``[B, kv_heads, T, dim]`` (a view)."""
        return store.view(store.size(0), store.size(2), self.kv_heads, dim).transpose(1, 2)

    def _sink(self, like: Tensor) -> Optional[Tensor]:
        if not self.sink:
            return None
        table = self.__dict__.setdefault("_constant_tensors", {})
        key = ("sink", str(like.device), like.dtype)
        if key not in table:
            table[key] = torch.zeros(self.heads, dtype=like.dtype, device=like.device)
        return table[key]

    def _kernels(self, p, values, batch, s, layer_id, cache, keep, positions, freq, sink, gate, mask) -> Tensor:
        """Norms, rotation and cache append in one launch, then the prompt or the decode kernel on the cached keys."""
        from ..ops import cuda_ops
        q = p["q"]
        holder = cache if cache is not None else StaticKVCache(s)
        wide = self.talk is not None
        sizes = (1, self.kv_heads * self.dim, self.kv_heads * self.vdim) if wide else (self.kv_heads, self.dim, self.vdim)
        ks, vs = holder.kv_storage(layer_id, batch, *sizes, q.dtype, q.device, s)
        wq, wk = (None, None) if self.q_norm is None else (self.q_norm.weight, self.k_norm.weight)
        if wide or self.halves or self.amplitude != 1.0:
            kh, vh = (self._heads(ks, self.dim), self._heads(vs, self.vdim)) if wide else (ks, vs)
            q = cuda_ops.head_prep(q, p["k"], values, wq, wk, self.eps, positions, freq, self.halves, self.amplitude, self.talk, kh, vh,
                                   holder.lengths_dev)
            vs = vh
        else:
            q = cuda_ops.qkv_prep(q, p["k"], values, wq, wk, self.eps, positions, freq, ks, vs, holder.lengths_dev)
        if s == 1 and cache is not None:
            return cuda_ops.grouped_decode(q[:, 0], ks, vs, holder.lengths_next, keep, sink, self.scale, self.softcap, gate, *mask)
        end = holder.length + s
        return cuda_ops.sink_attention(q, ks[:, :, :end].transpose(1, 2), vs[:, :, :end].transpose(1, 2), keep, sink, gate, self.scale,
                                       self.softcap, *mask)


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


class MatrixMemory(nn.Module):
    """mLSTM: per head a matrix memory ``S`` and a normaliser ``n`` with one input gate and one forget gate per token in the exponent,
    ``cap`` bounding both, and a running maximum that keeps them in range (``reference.matrix_memory``). A head's ``S^T q`` is divided by
    ``max(|n . q|, exp(-m)) + 1e-6`` and by its root mean square, then times a weight, times ``sigmoid(W_g h)``, and projected."""

    oslo_fused = False

    def __init__(self, width: int, heads: int, dim: int, vdim: int, cap: float, eps: float) -> None:
        super().__init__()
        self.heads, self.dim, self.vdim, self.cap, self.eps = heads, dim, vdim, float(cap), float(eps)
        self.in_proj = PackedLinear(width, {"q": heads * dim, "k": heads * dim, "v": heads * vdim, "g": heads * vdim})
        self.gates = Linear(width, 2 * heads)              # input gates, then forget gates; applied with 32-bit results
        self.o_norm = nn.Parameter(torch.ones(heads * vdim))
        self.out_proj = Linear(heads * vdim, width, bias=False)

    def forward(self, h: Tensor, batch: int, layer_id: int, cache: Optional[StaticKVCache], keep: Optional[Tensor]) -> MixerOutput:
        s = h.size(0) // batch
        keep = _last(keep, s)
        state = top = None
        if cache is not None:
            width = ops.reference.memory_state_width(self.vdim)
            state = cache.recurrent_state(layer_id, (batch, self.heads, self.dim, width), h.device)
            top = cache.recurrent_state(layer_id, (batch, self.heads), h.device, "max")
        p = self.in_proj(h)
        if s == 1 and state is not None and self.oslo_fused and _inference(h, self.o_norm) and ops.use_kernels(h):
            from ..ops import cuda_ops
            o = cuda_ops.memory_step(p["q"], p["k"], p["v"], h, self.gates.weight, self.gates.bias, self.cap, p["g"], self.o_norm, keep,
                                     state, top, self.eps, self.heads)
            return MixerOutput(self.out_proj(o), {})
        z = ops.linear_fp32(h, self.gates.weight, fused=self.oslo_fused)
        o, n, m = ops.matrix_memory(p["q"], p["k"], p["v"], z, self.gates.bias, self.cap, keep, state, top, batch, self.heads,
                                    fused=self.oslo_fused)
        o = ops.gated_rms_norm(o, self.o_norm, p["g"], self.eps, self.vdim, "sigmoid", (n, m), fused=self.oslo_fused)
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
        x = ops.causal_conv(p["x"], self.conv_weight, self.conv_bias, batch, keep, prev, silu=True, fused=self.oslo_fused)
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


class DenseMLP(nn.Module):
    """``W_down act(W_up h)``, ``act`` ``"relu2"`` (the square of relu) or a GeLU."""

    oslo_fused = False

    def __init__(self, width: int, ff: int, act: str = "relu2") -> None:
        super().__init__()
        self.act = act
        self.up = Linear(width, ff, bias=False)
        self.down = Linear(ff, width, bias=False)

    def forward(self, h: Tensor) -> FeedForwardOutput:
        return FeedForwardOutput(self.down(self.up(h, self.act)), {})


class MixtureOfExperts(nn.Module):
    """``experts`` small feed-forwards, of which a token uses ``top``. No capacity limit: every choice is computed. The result keeps one
    row per (token, choice); whoever adds it to the residual stream sums the rows.

    ``unit="relu2"``: ``W_down relu(W_up h)^2``; ``"silu"``: ``W_down (silu(W_gate h) * W_up h)``; ``"clamped"``: ``GatedMLP``'s unit with
    ``limit`` and ``alpha``. The router's logits are fp32: ``W_r h + b`` choose, weighted by the softmax over the chosen ones; ``scored``:
    scores are the softmax of ``W_r h`` over all outputs, ``score + correction`` choose, the weights are the chosen scores divided by
    their sum; ``scored="sigmoid"``: the largest ``sigmoid(W_r h)`` choose and are the weights as they are. ``identity`` further router
    outputs stand for the input itself. ``scale_input``: a weight multiplies what its expert reads, and the rows are summed without
    weights. ``shared``: size of an expert that every token uses, weighted by a sigmoid projection of its own (``shared_gate=False``:
    added as it is), with ``shared_limit`` where it is clamped."""

    oslo_fused = False

    def __init__(self, width: int, ff: int, experts: int, top: int, side: Optional[Dict[str, int]] = None, unit: str = "relu2",
                 scored=False, identity: int = 0, shared: Optional[int] = None, limit: float = 0.0, alpha: float = 1.702,
                 scale_input: bool = False, shared_gate: bool = True, shared_limit: Optional[float] = None) -> None:
        super().__init__()
        if unit not in ("relu2", "silu", "clamped"):
            raise ValueError(f"unknown expert unit {unit!r}")
        if scored not in (False, True, "sigmoid"):
            raise ValueError(f"unknown scores {scored!r}")
        self.experts, self.top, self.unit, self.scored, self.identity = experts, top, unit, scored, identity
        self.limit, self.alpha, self.scale_input, self.shared_gate = float(limit), float(alpha), bool(scale_input), bool(shared_gate)
        self.side = dict(side or {})
        self.in_proj = PackedLinear(width, self.side) if self.side else None
        outputs = experts + identity
        self.router = Linear(width, outputs, bias=not scored)
        self.correction = nn.Parameter(torch.zeros(outputs)) if scored is True else None
        self.up = nn.Parameter(torch.empty(experts, ff * (1 if unit == "relu2" else 2), width).normal_(std=0.02))
        self.down = nn.Parameter(torch.empty(experts, width, ff).normal_(std=0.02))
        self.shared = None
        if shared is not None:
            self.shared = GatedMLP(width, shared, side={"sg": 1} if shared_gate else None, limit=shared_limit, alpha=alpha)

    @staticmethod
    def interleave(gate: Tensor, up: Tensor) -> Tensor:
        """``up`` of a gated expert from its two matrices ``[ff, width]``: rows in turns, so that one tile holds both factors."""
        return torch.stack([gate, up], dim=1).reshape(2 * gate.size(0), gate.size(1))

    def forward(self, h: Tensor) -> FeedForwardOutput:
        side = self.in_proj(h) if self.in_proj is not None else {}
        bias = self.correction if self.scored else self.router.bias
        idx, weights = ops.moe_route(h, self.router.weight, bias, self.top, self.scored, fused=self.oslo_fused)
        y, slots = ops.moe_experts(h, idx, self.up, self.down, self.unit, self.limit, self.alpha, weights if self.scale_input else None,
                                   fused=self.oslo_fused)
        shared, gate = None, None
        if self.shared is not None:
            out = self.shared(h)
            shared, gate = out.y, out.side.get("sg")
        return FeedForwardOutput(y, side, slots, None if self.scale_input else weights, idx if self.identity else None, shared, gate)


class InputConvolution(nn.Module):
    """What a mixer reads is its input plus a causal convolution of it over time, per channel and without a bias: ``h + conv(h)``. The
    last ``taps - 1`` inputs are part of a sequence's state."""

    oslo_fused = False

    def __init__(self, width: int, taps: int) -> None:
        super().__init__()
        self.taps = taps
        self.weight = nn.Parameter(torch.empty(width, taps).normal_(std=taps ** -0.5))

    def state(self, batch: int, layer_id: int, cache: Optional[StaticKVCache], device) -> Optional[Tensor]:
        if cache is None:
            return None
        return cache.recurrent_state(layer_id, (batch, self.taps - 1, self.weight.size(0)), device, "inputs")

    def step(self, batch: int, layer_id: int, cache: Optional[StaticKVCache], keep: Optional[Tensor], device):
        """What the join kernel needs to do the convolution of single tokens on its way (``conv`` of ``cuda_ops.branch_join``)."""
        return self.weight, self.state(batch, layer_id, cache, device), _last(keep, 1)

    def forward(self, h: Tensor, batch: int, layer_id: int, cache: Optional[StaticKVCache], keep: Optional[Tensor]) -> Tensor:
        s = h.size(0) // batch
        return ops.causal_conv(h, self.weight, None, batch, _last(keep, s), self.state(batch, layer_id, cache, h.device), residual=True,
                               fused=self.oslo_fused)


class TokenInput(nn.Module):
    """A layer's input from the token itself: ``norm(W_proj (gelu(W_gate x) * e))`` with ``e`` the columns ``first`` to ``first + dim`` of the
    token's row of a table that the model's layers share. The result is a ``Branch`` of the residual stream ``x``."""

    oslo_fused = False

    def __init__(self, width: int, dim: int, first: int, eps: float) -> None:
        super().__init__()
        self.first = first
        self.gate = Linear(width, dim, bias=False)
        self.proj = Linear(dim, width, bias=False)
        self.norm = RMSNorm(width, eps)

    def forward(self, x: Tensor, ids: Tensor, table: Tensor) -> Branch:
        """``x`` ``[rows, width]`` in the weights' dtype, ``ids`` ``[rows]``, ``table`` ``[vocab, *]``."""
        return Branch(self.proj(ops.token_gate(self.gate(x), ids, table, self.first, fused=self.oslo_fused)), self.norm.weight)


class HyperConnections(nn.Module):
    """What ties one sublayer to ``streams`` residual streams: it reads ``sum_s w_in[s] x_s``; afterwards ``x_t <- sum_s mix[s, t] x_s +
    w_out[t] y`` (``reference.hyper_join``)."""

    oslo_fused = False

    def __init__(self, streams: int) -> None:
        super().__init__()
        self.w_in = nn.Parameter(torch.full((streams,), 1.0 / streams))
        self.w_out = nn.Parameter(torch.ones(streams))
        self.mix = nn.Parameter(torch.eye(streams))

    def forward(self, x: Tensor, result: Optional[ops.reference.SublayerResult], w_in: Optional[Tensor], norm: RMSNorm,
                scale: float = 1.0) -> Tuple[Tensor, Tensor]:
        """``x`` ``[rows, streams, width]`` with the sublayer's ``result``, and the input of the next sublayer, which reads with ``w_in``
        (``None``: the sum of the streams) through ``norm`` (weights around zero)."""
        return ops.hyper_join(x, result, self.w_out, self.mix, w_in, norm.weight, norm.eps, scale, fused=self.oslo_fused)
