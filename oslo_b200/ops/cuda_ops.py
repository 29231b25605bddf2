"""Autograd wrappers around the sm_100a kernels (``torch.ops.oslo_b200``).

Every function here assumes CUDA tensors; ``oslo_b200.ops.functional`` routes CPU tensors to the
PyTorch statements instead. GEMM operand layouts (see ``csrc/gemm_sm100.cu``): ``a_mn`` / ``b_mn`` say
that the operand is stored with the contraction dim as rows, which lets forward, dgrad and wgrad of
both weight layouts run without a transpose copy.
"""
from __future__ import annotations

import itertools
import os
from typing import Optional

import torch
from torch import Tensor

from . import load_ext
from ..config import get_config as _get_config
from . import reference as ref

FLAG_BIAS, FLAG_GELU, FLAG_SAVE_PREACT, FLAG_DGELU, FLAG_RESIDUAL, FLAG_OUT_FP32, FLAG_ACCUMULATE = 1, 2, 4, 8, 16, 32, 64
FLAG_RELU2, ACT_RELU2 = 1024, -2   # square of relu: in a GEMM's epilogue; as `gelu_from` of the few-row products
_GELU = ("gelu", "gelu_new", "gelu_tanh", "gelu_pytorch_tanh")
_16BIT = (torch.bfloat16, torch.float16)
_dropout_calls = itertools.count()


class _CheckedOps:
    """Debug wrapper around the operator namespace (``OSLO_B200_DEBUG_SYNC=1``): every operator call is followed by a
    device synchronisation and a read of the per-device error word, so a kernel whose bounded wait ran out - or an
    asynchronous CUDA error - is reported at the call that caused it, with the operator's name, instead of at some
    later synchronisation point. The reference has nothing comparable (its kernels never wait on each other)."""

    def __init__(self, ext) -> None:
        self._ext = ext

    def __getattr__(self, name):
        fn = getattr(self._ext, name)
        if name in ("error_word", "launch_count"):
            return fn

        def checked(*args, **kwargs):
            out = fn(*args, **kwargs)
            if torch.cuda.is_current_stream_capturing():
                return out
            torch.cuda.synchronize()
            like = next((a for a in args if isinstance(a, Tensor) and a.is_cuda), None)
            if like is not None:
                code = int(self._ext.error_word(like).item())
                if code:
                    self._ext.error_word(like).zero_()
                    raise RuntimeError(f"oslo_b200 kernel behind `{name}` gave up a bounded wait (device error code {code})")
            return out

        return checked


_CHECKED = None


def _ext():
    ext = load_ext(required=True)
    if _get_config().debug_sync:
        global _CHECKED
        if _CHECKED is None or _CHECKED._ext is not ext:
            _CHECKED = _CheckedOps(ext)
        return _CHECKED
    return ext


def device_error_code(like: Tensor) -> int:
    """Code left by a kernel whose bounded wait ran out (0 = none). Synchronises the device."""
    return int(_ext().error_word(like).item())


def reset_device_error(like: Tensor) -> None:
    _ext().error_word(like).zero_()


def _as_operand(t: Tensor) -> Tensor:
    """2-D tensor with contiguous last dim, 16-byte aligned rows."""
    if t.stride(-1) != 1 or t.stride(0) % 8 or t.data_ptr() % 16 or t.stride(0) < t.size(1):
        t = t.contiguous()
    return t


def gemm_ok(*ts: Tensor) -> bool:
    return all(t.dtype in _16BIT and t.size(-1) % 8 == 0 and t.size(0) > 0 for t in ts)


def gemm(a: Tensor, b: Tensor, a_mn: bool = False, b_mn: bool = False, bias: Optional[Tensor] = None,
         aux: Optional[Tensor] = None, out: Optional[Tensor] = None, aux_out: Optional[Tensor] = None,
         flags: int = 0, alpha: float = 1.0) -> Tensor:
    return _ext().gemm(_as_operand(a), _as_operand(b), int(a_mn), int(b_mn), bias, aux, out, aux_out, flags, alpha)


def gemm_nn(d: Tensor, w: Tensor) -> Tensor:
    """``d [n, V] @ w [V, H] -> [n, H]``."""
    return gemm(d, w, False, True)


def gemm_tn(d: Tensor, x: Tensor, out_dtype=None) -> Tensor:
    """``d[n, V].T @ x[n, H] -> [V, H]`` (fp32 output when ``out_dtype`` is float32)."""
    return gemm(d, x, True, True, flags=FLAG_OUT_FP32 if out_dtype == torch.float32 else 0)


SMALL_M_ROWS = 64  # inference calls with at most this many rows use the split-K path
GEMV_ROWS = 4      # ... and with at most this many rows the CUDA-core weight-streaming kernel


def weight_grad(weight: Tensor, a: Tensor, b: Tensor) -> Optional[Tensor]:
    """``a^T b`` (both ``[rows, *]``) as the gradient of ``weight``.

    Parameters whose ``.grad`` is a persistent, zeroed-per-step view of a flat buffer (marked
    ``_oslo_accum_grad`` by ``optim.FlatBuffers``) get the product accumulated into that view by the GEMM
    epilogue and ``None`` is returned, which spares the separate gradient tensor and the add kernel of every
    micro-batch; ``_oslo_grad_hook`` (set by the data-parallel wrapper) stands in for the post-accumulate hook
    that autograd does not call in that case."""
    g = weight.grad
    if (g is not None and getattr(weight, "_oslo_accum_grad", False) and g.dtype == weight.dtype
            and g.shape == weight.shape and g.is_contiguous() and not torch.is_grad_enabled()):
        gemm(a, b, True, True, out=g, flags=FLAG_ACCUMULATE)
        hook = getattr(weight, "_oslo_grad_hook", None)
        if hook is not None:
            hook(weight)
        return None
    return gemm(a, b, True, True)


class _Linear(torch.autograd.Function):
    @staticmethod
    def forward(ctx, x, weight, bias, reversed_, gelu, residual=None):
        k = x.size(-1)
        x2 = x.reshape(-1, k)
        need_grad = any(ctx.needs_input_grad[:3])  # grad mode is always off inside forward(); ask the ctx
        flags = (FLAG_BIAS if bias is not None else 0) | (FLAG_GELU if gelu else 0)
        n = weight.size(1) if reversed_ else weight.size(0)
        res2 = None
        if residual is not None:   # y = x W^T + b + residual in the GEMM epilogue (no activation in between)
            flags |= FLAG_RESIDUAL
            res2 = residual.reshape(-1, n)
            if res2.stride(-1) != 1:
                res2 = res2.contiguous()
        z = None
        if gelu and need_grad:
            flags |= FLAG_SAVE_PREACT
            z = torch.empty(x2.size(0), n, dtype=x.dtype, device=x.device)
        # the result is allocated in its final shape and the GEMM writes through a 2-D view of it: a view RETURNED by
        # a custom function could not be modified in place afterwards (the in-place rotary does that to q and k)
        y = torch.empty(*x.shape[:-1], n, dtype=x.dtype, device=x.device)
        gemm(x2, weight, False, reversed_, bias=bias, aux=res2, out=y.view(-1, n), aux_out=z, flags=flags)
        ctx.save_for_backward(x2, weight, z)
        ctx.reversed, ctx.has_bias, ctx.in_shape = reversed_, bias is not None, x.shape
        ctx.has_residual = residual is not None
        ctx.bias_dtype = bias.dtype if bias is not None else None
        return y

    @staticmethod
    def backward(ctx, dy):
        x2, weight, z = ctx.saved_tensors
        ext = _ext()
        dy2 = dy.reshape(-1, dy.size(-1))
        if not dy2.is_contiguous():
            dy2 = dy2.contiguous()
        if z is not None:
            dy2 = ext.bias_gelu_bwd(dy2, z, None)
        dx = dw = db = None
        if ctx.needs_input_grad[0]:
            dx = gemm(dy2, weight, False, not ctx.reversed).view(ctx.in_shape)
        if ctx.needs_input_grad[1]:
            dw = weight_grad(weight, x2, dy2) if ctx.reversed else weight_grad(weight, dy2, x2)
        if ctx.has_bias and ctx.needs_input_grad[2]:
            db = ext.colsum(dy2).to(ctx.bias_dtype)
        d_res = dy if (ctx.has_residual and ctx.needs_input_grad[5]) else None
        return dx, dw, db, None, None, d_res


class _FusedMLP(torch.autograd.Function):
    """``fc_out(gelu(fc_in(x)))`` for ``[out, in]`` weights. The backward multiplies by ``gelu'`` inside the epilogue
    of fc_out's input-gradient GEMM instead of running a separate pass over the ``[rows, 4 * hidden]`` activation
    gradient."""

    @staticmethod
    def forward(ctx, x, w_in, b_in, w_out, b_out, residual=None):
        k = x.size(-1)
        x2 = x.reshape(-1, k)
        need_grad = any(ctx.needs_input_grad)
        flags = FLAG_GELU | (FLAG_BIAS if b_in is not None else 0)
        z = None
        if need_grad:
            flags |= FLAG_SAVE_PREACT
            z = torch.empty(x2.size(0), w_in.size(0), dtype=x.dtype, device=x.device)
        h = gemm(x2, w_in, False, False, bias=b_in, aux_out=z, flags=flags)
        y = torch.empty(*x.shape[:-1], w_out.size(0), dtype=x.dtype, device=x.device)
        res2 = None
        if residual is not None:
            res2 = residual.reshape(-1, w_out.size(0))
            if res2.stride(-1) != 1:
                res2 = res2.contiguous()
        gemm(h, w_out, False, False, bias=b_out, aux=res2, out=y.view(-1, w_out.size(0)),
             flags=(FLAG_BIAS if b_out is not None else 0) | (FLAG_RESIDUAL if residual is not None else 0))
        ctx.save_for_backward(x2, w_in, w_out, z, h)
        ctx.has_b_in, ctx.has_b_out, ctx.in_shape = b_in is not None, b_out is not None, x.shape
        ctx.has_residual = residual is not None
        return y

    @staticmethod
    def backward(ctx, dy):
        x2, w_in, w_out, z, h = ctx.saved_tensors
        ext = _ext()
        dy2 = dy.reshape(-1, dy.size(-1))
        if not dy2.is_contiguous():
            dy2 = dy2.contiguous()
        dx = dw_in = db_in = dw_out = db_out = None
        dz = gemm(dy2, w_out, False, True, aux=z, flags=FLAG_DGELU)      # (dy W_out) * gelu'(z)
        if ctx.needs_input_grad[3]:
            dw_out = weight_grad(w_out, dy2, h)
        if ctx.has_b_out and ctx.needs_input_grad[4]:
            db_out = ext.colsum(dy2).to(dy.dtype)
        if ctx.needs_input_grad[0]:
            dx = gemm(dz, w_in, False, True).view(ctx.in_shape)
        if ctx.needs_input_grad[1]:
            dw_in = weight_grad(w_in, dz, x2)
        if ctx.has_b_in and ctx.needs_input_grad[2]:
            db_in = ext.colsum(dz).to(dy.dtype)
        d_res = dy if (ctx.has_residual and ctx.needs_input_grad[5]) else None
        return dx, dw_in, db_in, dw_out, db_out, d_res


def fused_mlp_ok(x: Tensor, w_in: Tensor, w_out: Tensor) -> bool:
    return (x.is_cuda and x.dtype in _16BIT and w_in.dtype == x.dtype and w_out.dtype == x.dtype and x.numel() > 0
            and x.size(-1) % 8 == 0 and w_in.size(0) % 8 == 0 and w_out.size(0) % 8 == 0
            and x.numel() // x.size(-1) > SMALL_M_ROWS)


def fused_mlp(x: Tensor, w_in: Tensor, b_in: Optional[Tensor], w_out: Tensor, b_out: Optional[Tensor],
              residual: Optional[Tensor] = None) -> Tensor:
    """``fc_out(gelu(fc_in(x))) (+ residual)``; the residual is added in fc_out's GEMM epilogue."""
    return _FusedMLP.apply(x, w_in, b_in, w_out, b_out, residual)


class _QKVLinear(torch.autograd.Function):
    """Three bias-free ``[out, in]`` projections of the same input. Forward is three GEMMs; the point is the
    backward: the three input-gradient GEMMs accumulate into one tensor in their epilogues instead of leaving two
    ``[rows, hidden]`` additions to autograd."""

    @staticmethod
    def forward(ctx, x, wq, wk, wv):
        k = x.size(-1)
        x2 = x.reshape(-1, k)
        outs = []
        for w in (wq, wk, wv):
            y = torch.empty(*x.shape[:-1], w.size(0), dtype=x.dtype, device=x.device)
            gemm(x2, w, False, False, out=y.view(-1, w.size(0)))
            outs.append(y)
        ctx.save_for_backward(x2, wq, wk, wv)
        ctx.in_shape = x.shape
        return tuple(outs)

    @staticmethod
    def backward(ctx, dq, dk, dv):
        x2, wq, wk, wv = ctx.saved_tensors
        dx = None
        dws = [None, None, None]
        for i, (d, w) in enumerate(((dq, wq), (dk, wk), (dv, wv))):
            if d is None:
                continue
            d2 = d.reshape(-1, d.size(-1))
            if not d2.is_contiguous():
                d2 = d2.contiguous()
            if ctx.needs_input_grad[0]:
                if dx is None:
                    dx = gemm(d2, w, False, True)
                else:
                    gemm(d2, w, False, True, out=dx, flags=FLAG_ACCUMULATE)
            if ctx.needs_input_grad[1 + i]:
                dws[i] = weight_grad(w, d2, x2)
        return (dx.view(ctx.in_shape) if dx is not None else None, *dws)


def qkv_linear(x: Tensor, wq: Tensor, wk: Tensor, wv: Tensor):
    return _QKVLinear.apply(x, wq, wk, wv)


def qkv_linear_ok(x: Tensor, *ws: Tensor) -> bool:
    return (x.is_cuda and x.dtype in _16BIT and x.numel() > 0 and x.size(-1) % 8 == 0
            and x.numel() // x.size(-1) > SMALL_M_ROWS and all(w.dtype == x.dtype and w.size(0) % 8 == 0 for w in ws))


def linear(x: Tensor, weight: Tensor, bias: Optional[Tensor], reversed_: bool, activation: Optional[str],
           residual: Optional[Tensor] = None) -> Tensor:
    """``act(x W^T + b)``; ``residual`` (no activation) is added in the GEMM epilogue on the large-input path."""
    if residual is not None:
        n_ = weight.size(1) if reversed_ else weight.size(0)
        big = (activation is None and x.is_cuda and x.dtype in _16BIT and weight.dtype == x.dtype and residual.dtype == x.dtype
               and x.size(-1) % 8 == 0 and n_ % 8 == 0 and x.numel() // max(x.size(-1), 1) > SMALL_M_ROWS
               and (bias is None or bias.dtype == x.dtype))
        if big:
            return _Linear.apply(x, weight, bias, reversed_, False, residual)
        return linear(x, weight, bias, reversed_, activation) + residual
    if activation is not None and activation not in _GELU + ("relu2",):
        raise ValueError(f"unsupported fused activation {activation!r}")
    n = weight.size(1) if reversed_ else weight.size(0)
    ok = (x.dtype in _16BIT and weight.dtype == x.dtype and x.size(-1) % 8 == 0 and n % 8 == 0 and x.numel() > 0
          and (bias is None or bias.dtype == x.dtype))
    if not ok:  # fp32 or ragged shapes: library GEMM, same semantics
        return ref.linear(x, weight, bias, reversed_, activation)
    rows = x.numel() // x.size(-1)
    if rows <= SMALL_M_ROWS and not (torch.is_grad_enabled() and (x.requires_grad or weight.requires_grad)):
        # decode steps: weight-streaming split-K GEMM so that every SM pulls weights, not just N / 128 of them
        x2 = _as_operand(x.reshape(rows, x.size(-1)))
        gelu_from = -1 if activation is None else (ACT_RELU2 if activation == "relu2" else 0)
        if rows <= GEMV_ROWS and not reversed_ and n % 4 == 0:
            y = _ext().gemv_rows(x2, None, _as_operand(weight), bias, gelu_from)   # no tensor-core tile to pad
        else:
            y = _ext().gemm_small_m(x2, _as_operand(weight), int(reversed_), bias, gelu_from)
        return y.view(*x.shape[:-1], n)
    if activation == "relu2":
        if torch.is_grad_enabled() and (x.requires_grad or weight.requires_grad):      # no backward of its own
            return torch.relu(_Linear.apply(x, weight, bias, reversed_, False, None)).pow(2)
        flags = FLAG_RELU2 | (FLAG_BIAS if bias is not None else 0)
        return gemm(x.reshape(rows, x.size(-1)), weight, False, reversed_, bias=bias, flags=flags).view(*x.shape[:-1], n)
    return _Linear.apply(x, weight, bias, reversed_, activation is not None, None)


def small_m_ok(x: Tensor, *weights: Tensor) -> bool:
    """Whether an inference call with input ``x`` takes the few-row (decode) GEMM path."""
    if torch.is_grad_enabled() and (x.requires_grad or any(w.requires_grad for w in weights)):
        return False
    rows = x.numel() // max(x.size(-1), 1)
    return (x.is_cuda and x.dtype in _16BIT and 0 < rows <= SMALL_M_ROWS and x.size(-1) % 8 == 0
            and all(w.dtype == x.dtype and w.size(0) % 8 == 0 for w in weights))


def packed_linear_small_m(x: Tensor, weight: Tensor, bias: Optional[Tensor], gelu_from: int) -> Tensor:
    """``x @ weight^T + bias`` for a few rows with tanh-GeLU on output columns ``>= gelu_from`` (-1: none);
    ``weight`` is the row-wise concatenation of several ``[out_i, in]`` layers that share the input."""
    rows = x.numel() // x.size(-1)
    x2 = _as_operand(x.reshape(rows, x.size(-1)))
    if rows <= GEMV_ROWS and weight.size(0) % 4 == 0:
        y = _ext().gemv_rows(x2, None, _as_operand(weight), bias, int(gelu_from))
    else:
        y = _ext().gemm_small_m(x2, _as_operand(weight), 0, bias, int(gelu_from))
    return y.view(*x.shape[:-1], weight.size(0))


def gemv_two_inputs(x1: Tensor, x2: Tensor, weight: Tensor, bias: Optional[Tensor] = None,
                    residual: Optional[Tensor] = None) -> Tensor:
    """``[x1 | x2] @ weight^T (+ bias) (+ residual)`` for at most ``GEMV_ROWS`` rows without materialising the
    concatenation."""
    return _ext().gemv_rows(_as_operand(x1), _as_operand(x2), _as_operand(weight), bias, -1, residual)


def rotary_append(q: Tensor, k: Tensor, v: Tensor, k_cache: Tensor, v_cache: Tensor, lengths: Tensor,
                  write_index: Tensor, rotary_dim: int, base: float = 10000.0) -> Tensor:
    """Decode step: rotary on the new token's ``q``/``k`` (``[B, heads*D]`` row slices, position ``lengths[b]``),
    ``k``/``v`` written into the static caches at ``write_index[0]``; returns the rotated ``q`` as ``[B, heads, D]``."""
    return _ext().rotary_append(q, k, v, k_cache, v_cache, lengths, write_index, int(rotary_dim), float(base))


class _LayerNorm(torch.autograd.Function):
    @staticmethod
    def forward(ctx, x, w, b, eps):
        xc = x.contiguous()
        y, mean, rstd = _ext().layernorm_fwd(xc, w, b, eps)
        ctx.save_for_backward(xc, w, mean, rstd)
        ctx.has_bias = b is not None
        return y

    @staticmethod
    def backward(ctx, dy):
        xc, w, mean, rstd = ctx.saved_tensors
        dx, dw, db = _ext().layernorm_bwd(dy.contiguous(), xc, w, mean, rstd)
        return dx, dw, (db if ctx.has_bias else None), None


def layer_norm(x: Tensor, w: Tensor, b: Optional[Tensor], eps: float) -> Tensor:
    vec = 4 if x.dtype == torch.float32 else 8
    cols = x.size(-1)
    if x.dtype != w.dtype or cols % vec or cols // vec > 1024 or x.numel() == 0:
        return ref.layer_norm(x, w, b, eps)
    return _LayerNorm.apply(x, w, b, eps)


class _BiasGelu(torch.autograd.Function):
    @staticmethod
    def forward(ctx, x, bias):
        xc = x.contiguous()
        ctx.save_for_backward(xc, bias)
        return _ext().bias_gelu_fwd(xc, bias)

    @staticmethod
    def backward(ctx, dy):
        xc, bias = ctx.saved_tensors
        dx = _ext().bias_gelu_bwd(dy.contiguous(), xc, bias)
        db = None
        if bias is not None and ctx.needs_input_grad[1]:
            db = _ext().colsum(dx.view(-1, dx.size(-1))).to(bias.dtype)
        return dx, db


def bias_gelu(x: Tensor, bias: Optional[Tensor]) -> Tensor:
    vec = 4 if x.dtype == torch.float32 else 8
    if x.size(-1) % vec or (bias is not None and bias.dtype != x.dtype) or x.numel() == 0:
        return ref.bias_gelu(x, bias)
    return _BiasGelu.apply(x, bias)


class _BiasDropoutResidual(torch.autograd.Function):
    @staticmethod
    def forward(ctx, x, bias, residual, p, seed):
        ctx.p, ctx.seed = p, seed
        ctx.has_bias, ctx.has_res = bias is not None, residual is not None
        ctx.bias_dtype = bias.dtype if bias is not None else None
        r = residual.contiguous() if residual is not None else None
        return _ext().bias_dropout_residual(x.contiguous(), bias, r, p, seed, 0)

    @staticmethod
    def backward(ctx, dy):
        dy = dy.contiguous()
        dx = _ext().bias_dropout_residual(dy, None, None, ctx.p, ctx.seed, 1) if ctx.p > 0 else dy
        db = _ext().colsum(dx.view(-1, dx.size(-1))).to(ctx.bias_dtype) if ctx.has_bias else None
        return dx, db, (dy if ctx.has_res else None), None, None


def bias_dropout_residual(x: Tensor, bias: Optional[Tensor], residual: Optional[Tensor], p: float, training: bool) -> Tensor:
    vec = 4 if x.dtype == torch.float32 else 8
    p = float(p) if training else 0.0
    if x.size(-1) % vec or x.numel() == 0 or (bias is not None and bias.dtype != x.dtype) or \
            (residual is not None and (residual.dtype != x.dtype or residual.shape != x.shape)):
        return ref.bias_dropout_residual(x, bias, residual, p, training)
    # the mask is a hash of (seed, element index): the seed follows torch's seed and a call counter so that
    # tensor-parallel ranks, which run the same call sequence under one seed, drop the same elements
    seed = (torch.initial_seed() * 1000003 + next(_dropout_calls)) & 0x7FFFFFFFFFFFFFFF
    return _BiasDropoutResidual.apply(x, bias, residual, p, seed)


class _Rotary(torch.autograd.Function):
    @staticmethod
    def forward(ctx, x, positions, rotary_dim, base):
        ctx.save_for_backward(positions)
        ctx.rd, ctx.base = rotary_dim, base
        return _ext().rotary(x.contiguous(), positions, rotary_dim, base, False)

    @staticmethod
    def backward(ctx, dy):
        (positions,) = ctx.saved_tensors
        return _ext().rotary(dy.contiguous(), positions, ctx.rd, ctx.base, True), None, None, None


class _RotaryInplace(torch.autograd.Function):
    """Rotation of the first ``rotary_dim`` dims of every head, in place: the other dims (3/4 of a GPT-J head) are
    neither read nor written. The input is the fresh output of a projection that nothing else needs, and the
    incoming gradient is the attention kernel's own output, so both directions may overwrite their argument.
    ``x`` is any contiguous tensor laid out ``[tokens, heads, head_dim]`` in memory."""

    @staticmethod
    def forward(ctx, x, positions, heads, head_dim, rotary_dim, base):
        ctx.save_for_backward(positions)
        ctx.cfg = (heads, head_dim, rotary_dim, base)
        ctx.mark_dirty(x)
        _ext().rotary_(x, positions, heads, head_dim, rotary_dim, base, False)
        return x

    @staticmethod
    def backward(ctx, dy):
        (positions,) = ctx.saved_tensors
        heads, head_dim, rotary_dim, base = ctx.cfg
        if not dy.is_contiguous():
            dy = dy.contiguous()
        return _ext().rotary_(dy, positions, heads, head_dim, rotary_dim, base, True), None, None, None, None, None


def rotary_interleaved(x: Tensor, positions: Tensor, rotary_dim: int, base: float) -> Tensor:
    if positions.dim() == 1:
        positions = positions.unsqueeze(0).expand(x.size(0), -1)
    positions = positions.to(torch.long).contiguous()
    heads, head_dim = x.size(-2), x.size(-1)
    ok = (x.dim() == 4 and x.is_contiguous() and head_dim % 8 == 0 and rotary_dim % 8 == 0 and x.data_ptr() % 16 == 0
          and not x.is_leaf and os.environ.get("OSLO_B200_ROTARY_INPLACE", "1") != "0")
    if ok:
        target = x
        if x._is_view():
            # work on the tensor the view was taken from (typically the projection's [B, S, heads * head_dim] output):
            # autograd refuses in-place changes of views that a custom function returned, and a plain function output
            # needs no view bookkeeping at all
            base_t = x._base
            if (base_t is not None and base_t.is_contiguous() and base_t.numel() == x.numel()
                    and base_t.data_ptr() == x.data_ptr() and not base_t._is_view() and not base_t.is_leaf):
                target = base_t
            elif x.requires_grad:
                ok = False
        if ok:
            out = _RotaryInplace.apply(target, positions, heads, head_dim, rotary_dim, base)
            return out if target is x else out.view(x.shape)
    return _Rotary.apply(x, positions, rotary_dim, base)


def flash_supported(q: Tensor, k: Tensor, v: Tensor) -> bool:
    if q.dtype not in _16BIT or q.size(-1) not in (64, 128, 256) or q.numel() == 0:
        return False
    return q.dtype == k.dtype == v.dtype


def _flash_impl() -> int:
    """1 = tcgen05/TMEM forward kernel (default), 0 = the mma.sync kernel (``OSLO_B200_ATTN=mma``)."""
    return 0 if os.environ.get("OSLO_B200_ATTN", "tcgen05") == "mma" else 1


def _attn_operand(t: Tensor) -> Tensor:
    if t.stride(-1) != 1 or any(s % 8 for s in t.stride()[:-1]) or t.data_ptr() % 16:
        t = t.contiguous()
    return t


class _Flash(torch.autograd.Function):
    @staticmethod
    def forward(ctx, q, k, v, causal, window, scale, kpm):
        q, k, v = _attn_operand(q), _attn_operand(k), _attn_operand(v)
        o, lse = _ext().flash_fwd(q, k, v, scale, causal, window, kpm, _flash_impl())
        ctx.save_for_backward(q, k, v, o, lse, kpm)
        ctx.cfg = (scale, causal, window)
        return o

    @staticmethod
    def backward(ctx, do):
        q, k, v, o, lse, kpm = ctx.saved_tensors
        scale, causal, window = ctx.cfg
        dq, dk, dv = _ext().flash_bwd(_attn_operand(do), q, k, v, o, lse, scale, causal, window, kpm, _flash_impl())
        return dq, dk, dv, None, None, None, None


def flash_attention(q: Tensor, k: Tensor, v: Tensor, causal: bool, window: Optional[int], scale: float,
                    key_padding_mask: Optional[Tensor]) -> Tensor:
    kpm = None
    if key_padding_mask is not None:
        kpm = (key_padding_mask != 0).to(torch.uint8).contiguous()
    return _Flash.apply(q, k, v, bool(causal), int(window or 0), float(scale), kpm)


def decode_attention(q: Tensor, k_cache: Tensor, v_cache: Tensor, lengths: Tensor, scale: float,
                     window: Optional[int]) -> Tensor:
    return _ext().decode_attn(q.contiguous(), k_cache, v_cache, lengths.to(torch.int32), float(scale), int(window or 0))


class _CausalSoftmax(torch.autograd.Function):
    @staticmethod
    def forward(ctx, x, scale):
        y = _ext().causal_softmax_fwd(x.contiguous(), scale)
        ctx.save_for_backward(y)
        ctx.scale = scale
        return y

    @staticmethod
    def backward(ctx, dy):
        (y,) = ctx.saved_tensors
        return _ext().softmax_bwd(y, dy.contiguous(), ctx.scale), None


def causal_softmax(x: Tensor, scale: float) -> Tensor:
    return _CausalSoftmax.apply(x, float(scale))


class _MaskedSoftmax(torch.autograd.Function):
    @staticmethod
    def forward(ctx, x, mask, scale):
        y = _ext().masked_softmax_fwd(x.contiguous(), mask, scale)
        ctx.save_for_backward(y)
        ctx.scale = scale
        return y

    @staticmethod
    def backward(ctx, dy):
        (y,) = ctx.saved_tensors
        return _ext().softmax_bwd(y, dy.contiguous(), ctx.scale), None, None


def masked_softmax(x: Tensor, mask: Tensor, scale: float) -> Tensor:
    return _MaskedSoftmax.apply(x, mask.to(torch.uint8).contiguous(), float(scale))


def ce_stats(logits: Tensor, labels: Tensor, vocab_start: int):
    return _ext().ce_stats(logits, labels.contiguous(), int(vocab_start))


def ce_grad_(logits: Tensor, labels: Tensor, vocab_start: int, lse: Tensor, scale: Tensor) -> Tensor:
    return _ext().ce_grad_(logits, labels.contiguous(), int(vocab_start), lse.contiguous(), scale.contiguous())


class _CrossEntropy(torch.autograd.Function):
    @staticmethod
    def forward(ctx, logits, labels, ignore_index):
        lg = logits if logits.stride(-1) == 1 else logits.contiguous()
        mx, se, tg = ce_stats(lg, labels, 0)
        lse = torch.log(se) + mx
        valid = labels != ignore_index
        count = valid.sum().clamp(min=1).to(torch.float32)
        ctx.save_for_backward(lg, labels, lse, valid, count)
        return torch.where(valid, lse - tg, torch.zeros_like(lse)).sum() / count

    @staticmethod
    def backward(ctx, g):
        lg, labels, lse, valid, count = ctx.saved_tensors
        scale = (g.float() / count) * valid.to(torch.float32)
        return ce_grad_(lg.clone(), labels, 0, lse, scale), None, None


def cross_entropy(logits: Tensor, labels: Tensor, ignore_index: int) -> Tensor:
    if logits.dim() != 2 or logits.dtype not in (torch.bfloat16, torch.float16, torch.float32):
        return ref.cross_entropy(logits, labels, ignore_index)
    return _CrossEntropy.apply(logits, labels, ignore_index)


def linear_cross_entropy(hidden: Tensor, weight: Tensor, bias: Optional[Tensor], labels: Tensor, ignore_index: int,
                         chunk_rows: int) -> Tensor:
    from ..parallel.vocab_parallel import linear_cross_entropy as lce
    fused = hidden.dtype in _16BIT and weight.dtype == hidden.dtype and hidden.size(-1) % 8 == 0 \
        and weight.size(0) % 8 == 0
    return lce(hidden, weight, bias, labels, ignore_index, chunk_rows, fused=fused)


def ban_repeated_ngrams(tokens: Tensor, lprobs: Tensor, n: int) -> Tensor:
    if lprobs.dtype != torch.float32 or not lprobs.is_contiguous():
        return ref.ban_repeated_ngrams(tokens, lprobs, n)
    return _ext().ngram_ban_(tokens.to(torch.long).contiguous(), lprobs, int(n))


# ---------------------------------------------------------------------------------------------------------------
# RMS norms, residual joins, gated recurrence, latent attention, mixture of experts (forward only)
def _rows(t: Tensor) -> Tensor:
    return t if t.stride(-1) == 1 else t.contiguous()


def _keep8(keep: Optional[Tensor]) -> Optional[Tensor]:
    if keep is None or keep.dtype == torch.uint8:
        return keep
    return (keep != 0).to(torch.uint8)


def rms_norm(x: Tensor, w: Tensor, eps: float, offset: float) -> Tensor:
    if x.dtype not in (w.dtype, torch.float32):
        x = x.to(w.dtype)
    return _ext().rms_norm(_rows(x.reshape(-1, x.size(-1))), w, float(eps), float(offset)).view(x.shape)


def residual_join(x: Tensor, y: Tensor, gate: Tensor, gate_bias: Tensor, w_post: Tensor, w_next: Optional[Tensor], eps: float,
                  slots: Optional[Tensor], slot_weights: Optional[Tensor]):
    xo, h = _ext().residual_join(x.contiguous(), _rows(y), slots, slot_weights, _rows(gate), gate_bias, w_post, w_next, float(eps))
    return xo, (h if w_next is not None else None)


def silu_mul(gate: Tensor, up: Tensor) -> Tensor:
    return _ext().silu_mul(_rows(gate), _rows(up))


RECURRENCE_MAX_DIM = 512   # key channels per head that one launch of the prompt kernel covers
BONUS_MAX_DIM = 256        # ... under the rule with a decay per channel
LATENT_MAX_RANK = 1024     # latent sizes that the decode kernel covers
GROUPED_MAX_VDIM = 1024    # value sizes that the grouped decode kernel covers
SINK_SMEM = 227 * 1024     # bytes of shared memory of a block of the 32-bit prompt kernel


def _channel_blocks(run, dim: int, limit: int, heads: int, state: Optional[Tensor], rows, vectors) -> Tensor:
    """``run(rows, vectors, state, dim)`` over blocks of at most ``limit`` key channels per head, outputs summed (key channels are
    independent of one another). ``rows`` ``[n, heads * dim]``, ``vectors`` ``[heads * dim]``."""
    if dim <= limit:
        return run(rows, vectors, state, dim)
    out = None
    for a in range(0, dim, limit):
        b = min(dim, a + limit)
        cut = lambda t: t.reshape(-1, heads, dim)[:, :, a:b].reshape(t.size(0), -1)            # noqa: E731
        part = state[:, :, a:b].contiguous() if state is not None else None
        o = run([cut(t) for t in rows], [cut(t[None])[0].contiguous() for t in vectors], part, b - a)
        if state is not None:
            state[:, :, a:b] = part
        out = o if out is None else out + o
    return out


def gated_recurrence(q: Tensor, f: Tensor, v: Tensor, f_bias: Tensor, lower: Tensor, norm_w: Tensor, eps: float, batch: int,
                     heads: int, keep: Optional[Tensor], state: Optional[Tensor]) -> Tensor:
    dim, vdim = q.size(1) // heads, v.size(1) // heads
    if q.size(0) == batch and state is not None:      # one token per sequence
        return _ext().recurrence_step(_rows(q), _rows(f), _rows(v), f_bias, lower, norm_w, _keep8(keep), state, float(eps), heads,
                                      dim, vdim)
    run = lambda r, w, s, d: _ext().recurrence(r[0], r[1], _rows(v), w[0], w[1], _keep8(keep), s, batch, heads, d, vdim)   # noqa: E731
    o = _channel_blocks(run, dim, RECURRENCE_MAX_DIM, heads, state, [_rows(q), _rows(f)], [f_bias, lower])
    return _ext().rms_norm(o.view(-1, vdim), norm_w, float(eps), 0.0).view(-1, heads * vdim)


def decayed_attention(q: Tensor, k: Tensor, v: Tensor, decay: Tensor, keep: Optional[Tensor], state: Optional[Tensor], batch: int,
                      heads: int) -> Tensor:
    dim, vdim = q.size(1) // heads, v.size(1) // heads
    q, k, v, keep = _rows(q), _rows(k), _rows(v), _keep8(keep)
    if q.size(0) == batch and state is not None:
        return _ext().decayed_step(q, k, v, decay, keep, state, heads, dim, vdim)
    run = lambda r, w, s, d: _ext().decayed_recurrence(r[0], r[1], v, decay, keep, s, batch, heads, d, vdim)                # noqa: E731
    return _channel_blocks(run, dim, RECURRENCE_MAX_DIM, heads, state, [q, k], []).view(q.size(0), -1)


def bonus_recurrence(r: Tensor, k: Tensor, v: Tensor, z: Tensor, w0: Tensor, u: Tensor, keep: Optional[Tensor],
                     state: Optional[Tensor], batch: int, heads: int) -> Tensor:
    dim, vdim = r.size(1) // heads, v.size(1) // heads
    v, keep = _rows(v), _keep8(keep)
    run = lambda x, w, s, d: _ext().bonus_recurrence(x[0], x[1], v, x[2], w[0], w[1], keep, s, batch, heads, d, vdim)       # noqa: E731
    return _channel_blocks(run, dim, BONUS_MAX_DIM, heads, state, [_rows(r), _rows(k), _rows(z)], [w0, u]).view(r.size(0), -1)


def bonus_step(r: Tensor, k: Tensor, v: Tensor, t: Tensor, w2: Tensor, w0: Tensor, u: Tensor, norm_w: Tensor, gate: Tensor,
               keep: Optional[Tensor], state: Tensor, eps: float, heads: int) -> Tensor:
    """Decode step: decay projection, recurrence, head norms and gate in one launch; ``t`` is ``W_w1 mix`` before its tanh."""
    return _ext().bonus_step(_rows(r), _rows(k), _rows(v), _rows(t), w2, w0, u, norm_w, _rows(gate), _keep8(keep), state, float(eps),
                             heads, r.size(1) // heads, v.size(1) // heads)


def linear_fp32(x: Tensor, weight: Tensor) -> Tensor:
    if gemm_ok(x, weight) and weight.dtype == x.dtype:
        n = weight.size(0)
        out = torch.empty(x.size(0), -(-n // 4) * 4, dtype=torch.float32, device=x.device)[:, :n]   # rows at 16-byte boundaries
        return gemm(x, weight, out=out, flags=FLAG_OUT_FP32)
    return torch.matmul(x.float(), weight.float().t())


def stacked_linear(x: Tensor, weight: Tensor):
    """A few rows: all parts' rows against all parts' weights in one weight-streaming product, of which the diagonal blocks are
    kept - reading the weights is what takes time there."""
    parts, rows, k = x.shape
    n = weight.size(1)
    if not (gemm_ok(x[0], weight[0]) and n % 8 == 0):
        return torch.matmul(x, weight.transpose(1, 2)).unbind(0)
    if rows <= GEMV_ROWS:
        return _ext().gemv_stacked(x, weight).unbind(0)
    if rows <= SMALL_M_ROWS and x.is_contiguous() and weight.is_contiguous():
        flat, w = x.view(parts * rows, k), weight.view(parts * n, k)
        y = _ext().gemm_small_m(flat, w, 0, None, -1) if parts * rows <= SMALL_M_ROWS else gemm(flat, w)
        return tuple(y[i * rows:(i + 1) * rows, i * n:(i + 1) * n] for i in range(parts))
    return tuple(gemm(x[i], weight[i]) for i in range(parts))


def branch_join(x: Tensor, branches, mult: float, eps: float, w_next, copy: Optional[torch.dtype] = None, conv=None):
    """``reference.branch_join``. ``conv`` ``(weight, state, keep)``, for rows that are single tokens: a second result, the first norm plus its
    causal convolution (``reference.causal_conv`` with ``residual``), whose state moves on."""
    bs = [ref.Branch(*b) for b in branches]
    w = list(w_next) + [None] * (2 - len(w_next))
    conv_w, state, keep = (None, None, None) if conv is None else conv
    xo, h1, h2, co = _ext().branch_join(x.contiguous(), [_rows(b.y) for b in bs], [b.weight for b in bs], [float(b.factor) for b in bs],
                                        [int(b.normed) for b in bs], [b.slots for b in bs], [int(b.top) for b in bs], float(mult),
                                        float(eps), w[0], w[1], copy is not None, conv_w, state, _keep8(keep))
    return xo, [h1, co] if conv is not None else [h1, h2][:1 if copy is not None else len(w_next)]


def token_gate(z: Tensor, ids: Tensor, table: Tensor, first: int) -> Tensor:
    return _ext().token_gate(_rows(z), ids.reshape(-1), table, int(first))


def clamped_glu(gate: Tensor, up: Tensor, limit: float, alpha: float) -> Tensor:
    return _ext().clamped_glu(_rows(gate), _rows(up), float(limit), float(alpha))


def gated_rms_norm(o: Tensor, w: Tensor, gate: Tensor, eps: float, group: int, act: str, normalizer=None) -> Tensor:
    z, m = (None, None) if normalizer is None else (t.contiguous() for t in normalizer)
    return _ext().gated_rms_norm(o.contiguous(), w, _rows(gate), float(eps), int(group), {"sigmoid": 0, "silu": 1}[act], z, m)


HYPER_MAX_TOP = 64     # rows per token that the stream join adds up
HYPER_MAX_STREAMS = 16


def hyper_join(x: Tensor, result, w_out: Optional[Tensor], mix: Optional[Tensor], w_in: Optional[Tensor], w_norm: Tensor, eps: float,
               scale: float):
    r = result if result is not None else ref.SublayerResult(None)
    if x.size(1) > HYPER_MAX_STREAMS or (r.weights is not None and r.weights.size(1) > HYPER_MAX_TOP):
        return ref.hyper_join(x, result, w_out, mix, w_in, w_norm, eps, scale)
    rows = lambda t: None if t is None else _rows(t)                                       # noqa: E731
    xo, h = _ext().hyper_join(x if x.stride(-1) == 1 else x.contiguous(), rows(r.y), r.slots, r.weights, r.choice, int(r.experts),
                              rows(r.h), rows(r.shared), rows(r.shared_gate), w_out, mix, w_in, w_norm, float(eps), float(scale))
    return (xo if result is not None else x), h


def matrix_memory(q: Tensor, k: Tensor, v: Tensor, z: Tensor, bias: Tensor, cap: float, keep: Optional[Tensor],
                  state: Optional[Tensor], top: Optional[Tensor], batch: int, heads: int):
    dim, vdim = q.size(1) // heads, v.size(1) // heads
    q, k, v, keep, scale = _rows(q), _rows(k), _rows(v), _keep8(keep), dim ** -0.5
    read, write, start, m = _ext().memory_gates(_rows(z), bias, float(cap), keep, top, batch)
    run = lambda a, b, s, d: _ext().memory_recurrence(a, b, v, read, write, start, scale, keep, s, batch, heads, d, vdim)   # noqa: E731
    if dim <= RECURRENCE_MAX_DIM:
        o, n = run(q, k, state, dim)
        return o, n, m
    o = n = 0.0                                            # key channels are independent of one another
    for a in range(0, dim, RECURRENCE_MAX_DIM):
        b = min(dim, a + RECURRENCE_MAX_DIM)
        cut = lambda t: t.reshape(-1, heads, dim)[:, :, a:b].reshape(t.size(0), -1)        # noqa: E731
        part = state[:, :, a:b].contiguous() if state is not None else None
        more_o, more_n = run(cut(q), cut(k), part, b - a)
        o, n = o + more_o, n + more_n
        if state is not None:
            state[:, :, a:b] = part
    return o, n, m


MEMORY_STEP_MAX = 46 * 1024 - 4096   # bytes of shared memory that a step's key channels may take


def memory_step(q: Tensor, k: Tensor, v: Tensor, x: Tensor, w: Tensor, bias: Tensor, cap: float, gate: Tensor, norm_w: Tensor,
                keep: Optional[Tensor], state: Tensor, top: Tensor, eps: float, heads: int) -> Tensor:
    """Decode step: gates from the mixer's input ``x``, memory, normaliser, head norms and output gate in one launch."""
    dim, vdim = q.size(1) // heads, v.size(1) // heads
    if 12 * dim > MEMORY_STEP_MAX:
        o, n, m = matrix_memory(q, k, v, linear_fp32(x, w), bias, cap, keep, state, top, q.size(0), heads)
        return gated_rms_norm(o, norm_w, gate, eps, vdim, "sigmoid", (n, m))
    return _ext().memory_step(_rows(q), _rows(k), _rows(v), _rows(x), w, bias, float(cap), _rows(gate), norm_w, _keep8(keep), state, top,
                              dim ** -0.5, float(eps), heads, dim, vdim)


def token_shift(h: Tensor, mu: Tensor, batch: int, keep: Optional[Tensor], prev: Optional[Tensor]) -> Tensor:
    return _ext().token_shift(_rows(h), mu, batch, _keep8(keep), prev)


def causal_conv(x: Tensor, w: Tensor, bias: Optional[Tensor], batch: int, keep: Optional[Tensor], prev: Optional[Tensor],
                silu: bool = False, residual: bool = False) -> Tensor:
    return _ext().causal_conv(_rows(x), w, bias, batch, _keep8(keep), prev, bool(silu), bool(residual))


SCAN_MAX_STATES = 256   # states per channel that one launch of the prompt scan covers


def selective_scan(x: Tensor, dt: Tensor, dt_bias: Tensor, a_log: Tensor, b: Tensor, c: Tensor, d: Tensor, z: Tensor, batch: int,
                   keep: Optional[Tensor], state: Optional[Tensor]) -> Tensor:
    if a_log.size(1) > SCAN_MAX_STATES:
        y, final = ref.selective_scan(x, dt, dt_bias, a_log, b, c, d, z, batch, keep, state)
        if state is not None:
            state.copy_(final)
        return y
    return _ext().selective_scan(_rows(x), _rows(dt), dt_bias, a_log, _rows(b), _rows(c), d, _rows(z), batch, _keep8(keep), state)


def scan_step(x: Tensor, dt: Tensor, w_dt: Tensor, dt_bias: Tensor, a_log: Tensor, b: Tensor, c: Tensor, d: Tensor, z: Tensor,
              keep: Optional[Tensor], state: Tensor) -> Tensor:
    """Decode step: step projection ``w_dt dt``, state update, gate in one launch."""
    return _ext().scan_step(_rows(x), _rows(dt), w_dt, dt_bias, a_log, _rows(b), _rows(c), d, _rows(z), _keep8(keep), state)


def qkv_prep(q: Tensor, k: Tensor, v: Tensor, wq: Optional[Tensor], wk: Optional[Tensor], eps: float, positions: Tensor, freq: Tensor,
             k_store: Tensor, v_store: Tensor, lengths: Tensor) -> Tensor:
    """Head norms (weights or ``None``) and rotation of queries and keys; keys and values go into the caches at ``lengths[row]``. Returns
    ``[B, S, H, dim]``."""
    return _ext().qkv_prep(_rows(q), _rows(k), _rows(v), wq, wk, float(eps), positions, freq, k_store, v_store, lengths)


def head_prep(q: Tensor, k: Tensor, v: Tensor, wq: Optional[Tensor], wk: Optional[Tensor], eps: float, positions: Tensor, freq: Tensor,
              halves: bool, amplitude: float, talk: Optional[Tensor], k_store: Tensor, v_store: Tensor, lengths: Tensor) -> Tensor:
    """``qkv_prep`` with either rotation, scaled sines and cosines, and caches of any strides ``[B, G, T, *]``. ``talk``: the queries of mixed
    scores instead (``reference.norm_rotate_fold``), ``[B, S, H, G * dim]``."""
    return _ext().head_prep(_rows(q), _rows(k), _rows(v), wq, wk, float(eps), positions, freq, bool(halves), float(amplitude), talk, k_store,
                            v_store, lengths)


def grouped_decode(q: Tensor, k: Tensor, v: Tensor, lengths: Tensor, keep: Optional[Tensor], sink: Optional[Tensor], scale: float,
                   softcap: float, gate: Optional[Tensor] = None, window: int = 0, keep_first: int = 0,
                   lead: Optional[Tensor] = None) -> Tensor:
    """``v`` may have more heads than ``k`` when ``k`` has one and ``v`` is a view of rows that hold all its heads."""
    heads = v.size(1) // k.size(1)
    if heads == 1:
        fits = v.size(-1) <= GROUPED_MAX_VDIM
    else:
        fits = _ext().wide_decode_fits(q, q.size(1), heads, k.size(-1), heads * v.size(-1))
    if not fits:
        return ref.grouped_decode(q, k, v, lengths, keep, sink, scale, softcap, gate, window, keep_first, lead)
    if heads > 1:
        v = v.transpose(1, 2).flatten(2).unsqueeze(1)      # a view again
    return _ext().grouped_decode(q.contiguous(), k, v, lengths, _keep8(keep), sink, float(scale), float(softcap),
                                 None if gate is None else _rows(gate), int(window), int(keep_first), lead, heads)


def flash_head_dim(dim: int, vdim: int) -> int:
    """Head size at which the tcgen05 flash kernel can run heads of ``dim`` / ``vdim`` (0: none)."""
    return next((d for d in (64, 128, 256) if d >= max(dim, vdim)), 0)


def pad_heads(t: Tensor, d: int) -> Tensor:
    """``[B, S, H, dim] -> [B, S, H, d]``, zero-padded (no copy when the size already fits)."""
    return t if t.size(-1) == d else torch.nn.functional.pad(t, (0, d - t.size(-1)))


def flash_parts_fit(dim: int, rot: int, vdim: int) -> bool:
    """Whether the tcgen05 flash kernel runs heads of ``dim`` + ``rot`` query and key dimensions from two operands."""
    return dim % 8 == 0 and rot % 8 == 0 and vdim % 8 == 0 and -(-dim // 64) + -(-rot // 64) <= 4 and vdim <= 256


def sink_attention(q: Tensor, k: Tensor, v: Tensor, keep: Optional[Tensor], sink: Optional[Tensor], gate: Optional[Tensor], scale: float,
                   softcap: float = 0.0, window: int = 0, keep_first: int = 0, lead: Optional[Tensor] = None,
                   q_rot: Optional[Tensor] = None, k_rot: Optional[Tensor] = None) -> Tensor:
    """``q`` ``[B, Sq, H, dim]``, ``k``/``v`` ``[B, Sk, G, *]`` (``k`` may have one head where ``v`` has several). 16-bit heads run on the tcgen05 flash kernel, with sink, gate, cap and
    window in its softmax and epilogue, and a second operand for the key part that heads share (gated value sizes that are no
    multiple of 8: zero-padded heads, sink and gate from its log-sum-exp); everything else in the fp32 kernel."""
    dim, vdim = q.size(-1), v.size(-1)
    d = flash_head_dim(dim, vdim)
    mask = (int(window), int(keep_first), lead)
    flash = q.dtype in _16BIT and d and q.size(1) > 1
    gate = None if gate is None else _rows(gate)
    if k.size(2) == 1 and (v.size(2) > 1 or not d):
        flash = False
        if q.dtype in _16BIT and q.size(1) > 1 and not softcap and q_rot is None and dim % 8 == 0 and vdim % 8 == 0 and vdim <= 256:
            if gate is not None and gate.size(1) != q.size(2):
                gate = _attn_operand(gate)                 # a gate per element is read in 16-byte pieces
            kpm = _keep8(keep).contiguous() if keep is not None else None
            qh, kh, vh = (_attn_operand(t.permute(0, 2, 1, 3)) for t in (q, k, v))
            return _ext().flash_wide_fwd(qh, kh, vh, kpm, sink, gate, float(scale), *mask)
    if flash and gate is not None and gate.size(1) != q.size(2):
        gate = _attn_operand(gate)                         # a gate per element is read in 16-byte pieces
    if q_rot is not None:
        if flash and not softcap and flash_parts_fit(dim, q_rot.size(-1), vdim):
            kpm = _keep8(keep).contiguous() if keep is not None else None
            qh, kh, vh, q2 = (_attn_operand(t.permute(0, 2, 1, 3)) for t in (q, k, v, q_rot))
            return _ext().flash_sink_fwd(qh, kh, vh, kpm, sink, gate, float(scale), 0.0, *mask, q2, _attn_operand(k_rot))
        q = torch.cat([q, q_rot], dim=-1)
        k = torch.cat([k, k_rot.unsqueeze(2).expand(-1, -1, k.size(2), -1)], dim=-1)
        return sink_attention(q, k, v, keep, sink, gate, scale, softcap, *mask)
    if flash:
        kpm = _keep8(keep).contiguous() if keep is not None else None
        if dim % 8 == 0 and vdim % 8 == 0:
            qh, kh, vh = (_attn_operand(t.permute(0, 2, 1, 3)) for t in (q, k, v))
            return _ext().flash_sink_fwd(qh, kh, vh, kpm, sink, gate, float(scale), float(softcap), *mask)
        if (gate is not None and sink is not None and gate.size(1) == q.size(2) and not softcap and not window
                and k.size(2) == q.size(2)):
            qh, kh, vh = (_attn_operand(pad_heads(t, d).permute(0, 2, 1, 3)) for t in (q, k, v))
            o, lse = _ext().flash_fwd(qh, kh, vh, float(scale), True, 0, kpm, _flash_impl())
            return _ext().sink_gate(o, lse, sink, gate, vdim)
    if 4 * (48 * (dim + vdim + 2) + 528) > SINK_SMEM:      # 16 queries and 32 keys and values of the kernel do not fit
        return ref.sink_attention(q, k, v, keep, sink, gate, scale, softcap, *mask)[0]
    return _ext().sink_attention(*(t if t.stride(-1) == 1 else t.contiguous() for t in (q, k, v)), _keep8(keep), sink, gate,
                                 float(scale), float(softcap), *mask)


def latent_prep(cq: Tensor, wq: Tensor, ckv: Optional[Tensor], wkv: Optional[Tensor], cache: Optional[Tensor], lengths: Tensor,
                eps: float, positions: Optional[Tensor] = None, freq: Optional[Tensor] = None, rows: bool = False):
    """The normed query latents; the normed key-value latents, and behind them what ``ckv`` has besides, rotated, go into ``cache`` at
    position ``lengths[row]`` and on. ``rows``: also the normed key-value latents as rows."""
    return _ext().latent_prep(_rows(cq), wq, None if ckv is None else _rows(ckv), wkv, cache, lengths, float(eps), positions, freq, rows)


def rotate_halves_(q: Tensor, positions: Tensor, freq: Tensor) -> Tensor:
    """The last ``2 * len(freq)`` dims of ``q`` ``[B, S, heads, dim]`` rotated in place."""
    return _ext().rotate_halves_(q, positions, freq)


def latent_decode(q: Tensor, w_uk: Tensor, w_uv: Tensor, cache: Tensor, lengths: Tensor, keep: Optional[Tensor],
                  sink: Optional[Tensor], gate: Tensor, scale: float, heads: int, positions: Optional[Tensor] = None,
                  freq: Optional[Tensor] = None) -> Tensor:
    return _ext().latent_decode(_rows(q), w_uk, w_uv, cache, lengths.to(torch.int32), _keep8(keep), sink, _rows(gate),
                                float(scale), heads, positions, freq)


MOE_UNITS = {None: 0, "relu2": 1, "silu": 2, "clamped": 3}
MOE_SCORES = {False: 0, True: 1, "sigmoid": 2}
MOE_FEW_PAIRS = 8   # (token, choice) pairs up to which the chosen experts' weights are streamed per pair


def moe_route(h: Tensor, w: Tensor, bias: Optional[Tensor], top: int, scored=False):
    logits = None
    if h.size(0) > SMALL_M_ROWS and gemm_ok(h, w):
        logits = linear_fp32(h, w)                         # 16-bit operands, exact products, fp32 sums and output
    elif h.size(0) > 65535:                                # no tensor-core path for these sizes or types: 32-bit library product
        logits = torch.matmul(h.float(), w.float().t())
    return _ext().moe_route(_rows(h), w, bias, logits, top, MOE_SCORES[scored])


def moe_experts(h: Tensor, idx: Tensor, up: Tensor, down: Tensor, unit: str = "relu2", limit: float = 0.0, alpha: float = 1.702,
                scale: Optional[Tensor] = None):
    u = MOE_UNITS[unit]
    if idx.numel() <= MOE_FEW_PAIRS:
        a = _ext().moe_few(_rows(h), idx, up, idx.size(1), u, float(limit), float(alpha), scale)
        return _ext().moe_few(a, idx, down, 1, 0), None
    slots, rows, tile_group, n_tiles = _ext().moe_plan(_rows(h), idx, up.size(0), scale)
    a = _ext().moe_grouped(rows, up, tile_group, n_tiles, u, float(limit), float(alpha))
    return _ext().moe_grouped(a, down, tile_group, n_tiles, 0), slots
