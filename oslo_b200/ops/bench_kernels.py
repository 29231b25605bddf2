"""Micro-benchmarks of the hand-written kernels against library baselines, timed with CUDA events.

``python -m oslo_b200.ops.bench_kernels --op gemm``       tcgen05 GEMM vs ``torch.matmul`` (cuBLAS), GPT-J shapes
``python -m oslo_b200.ops.bench_kernels --op attention``  tcgen05 flash attention (forward, backward) vs the
                                                           mma.sync kernels of this package
``python -m oslo_b200.ops.bench_kernels --op mixers``      the prompt and decode kernels of the recurrence, latent-attention,
                                                           expert and norm layers, each with its bound (HBM bytes, bf16
                                                           tensor-core or fp32 FMA throughput, whichever is slowest),
                                                           beside the like kernels of GPT-J at the same sizes
``python -m oslo_b200.ops.bench_kernels --op branches``    the same for grouped-query attention, the linear recurrences, the
                                                           selective scan and the branch joins, beside those
``python -m oslo_b200.ops.bench_kernels --op streams``     the same for windowed and two-part attention, matrix memory, gated and
                                                           identity experts and the stream join, beside those
``python -m oslo_b200.ops.bench_kernels --op talk``        the same for attention with mixed heads, clamped experts with scaled inputs,
                                                           input convolutions and per-token layer inputs, beside those
``--case i`` restricts the run to one shape and ``--iters n --warmup w`` bound the number of launches, which is
what a profiler capture wants. Every line is JSON; ``frac_of_measured`` divides by the bf16 GEMM throughput in
``MEASURED_PEAKS.json`` at the repository root when that file exists (else by 1590 TFLOP/s).

Timing: ``warmup`` untimed calls, then ``iters`` calls each bracketed by events on the launching stream with a
write of a 256 MB buffer in between (L2 flush); the median is reported.
"""
from __future__ import annotations

import argparse
import json
import math
import os

import torch

from . import cuda_ops as co
from . import load_ext

GEMM_CASES = [  # M, N, K, a_mn_major, b_mn_major
    (16384, 4096, 4096, 0, 0), (16384, 16384, 4096, 0, 0), (16384, 4096, 16384, 0, 0), (16384, 12288, 4096, 0, 0),
    (16384, 4096, 4096, 0, 1), (4096, 4096, 16384, 1, 1), (16384, 4096, 16384, 1, 1), (8192, 8192, 8192, 0, 0),
    (8192, 50400, 4096, 0, 0),
]
ATTN_CASES = [  # B, H, S, D
    (4, 16, 2048, 256), (4, 32, 2048, 128), (4, 32, 2048, 64), (1, 16, 8192, 256),
]


def _peak_tflops() -> float:
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    try:
        with open(path) as f:
            return float(json.load(f)["bf16_tflops"])
    except Exception:
        return 1590.0


class _Timer:
    def __init__(self, iters: int, warmup: int, flush: bool):
        self.iters, self.warmup = iters, warmup
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda") if flush else None

    def __call__(self, fn) -> float:
        for _ in range(self.warmup):
            fn()
        ts = []
        for _ in range(self.iters):
            if self.flush is not None:
                self.flush.zero_()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            ts.append(a.elapsed_time(b))
        ts.sort()
        return ts[len(ts) // 2]


class _GraphTimer(_Timer):
    """The same timing with ``fn`` captured once into a CUDA graph and replayed, which is how decode steps run: without the
    host's launch work, that takes longer than a small kernel."""

    def __call__(self, fn) -> float:
        side = torch.cuda.Stream()
        side.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(side):
            for _ in range(2):
                fn()
        torch.cuda.current_stream().wait_stream(side)
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            fn()
        ms = super().__call__(graph.replay)
        del graph
        return ms


def bench_gemm(args, timer: _Timer) -> None:
    peak = _peak_tflops()
    cases = GEMM_CASES if args.case is None else [GEMM_CASES[args.case]]
    for (M, N, K, amn, bmn) in cases:
        A = torch.randn(M, K, device="cuda", dtype=torch.bfloat16)
        B = torch.randn(N, K, device="cuda", dtype=torch.bfloat16)
        a = A.t().contiguous() if amn else A
        b = B.t().contiguous() if bmn else B
        t = timer(lambda: co.gemm(a, b, bool(amn), bool(bmn)))
        rec = dict(op="gemm", M=M, N=N, K=K, a_mn_major=amn, b_mn_major=bmn, ms=round(t, 4),
                   tflops=round(2.0 * M * N * K / t / 1e9, 1))
        rec["frac_of_measured"] = round(rec["tflops"] / peak, 3)
        if not args.no_baseline:
            tb = timer(lambda: torch.matmul(a.t() if amn else a, b if bmn else b.t()))
            rec.update(cublas_ms=round(tb, 4), cublas_tflops=round(2.0 * M * N * K / tb / 1e9, 1))
        print(json.dumps(rec), flush=True)


def bench_attention(args, timer: _Timer) -> None:
    ext = load_ext(required=True)
    peak = _peak_tflops()
    cases = ATTN_CASES if args.case is None else [ATTN_CASES[args.case]]
    for (B, H, S, D) in cases:
        mk = lambda: (torch.randn(B, S, H, D, device="cuda") * 0.5).to(torch.bfloat16).permute(0, 2, 1, 3)
        q, k, v, do = mk(), mk(), mk(), mk()
        sc = 1.0 / math.sqrt(D)
        for causal in ((True, False) if args.causal is None else (bool(args.causal),)):
            o, lse = ext.flash_fwd(q, k, v, sc, causal, 0, None, 1)
            frac = 0.5 if causal else 1.0
            fl_f, fl_b = 4.0 * B * H * S * S * D * frac, 10.0 * B * H * S * S * D * frac
            tf = timer(lambda: ext.flash_fwd(q, k, v, sc, causal, 0, None, 1))
            tb = timer(lambda: ext.flash_bwd(do, q, k, v, o, lse, sc, causal, 0, None, 1))
            rec = dict(op="attention", B=B, H=H, S=S, D=D, causal=causal, fwd_ms=round(tf, 4), bwd_ms=round(tb, 4),
                       fwd_tflops=round(fl_f / tf / 1e9, 1), bwd_tflops=round(fl_b / tb / 1e9, 1))
            rec["fwd_frac_of_measured"] = round(rec["fwd_tflops"] / peak, 3)
            rec["bwd_frac_of_measured"] = round(rec["bwd_tflops"] / peak, 3)
            if not args.no_baseline:
                tf0 = timer(lambda: ext.flash_fwd(q, k, v, sc, causal, 0, None, 0))
                tb0 = timer(lambda: ext.flash_bwd(do, q, k, v, o, lse, sc, causal, 0, None, 0))
                rec.update(mma_sync_fwd_ms=round(tf0, 4), mma_sync_bwd_ms=round(tb0, 4))
            rec["device_error_word"] = int(ext.error_word(q).item())
            print(json.dumps(rec), flush=True)


# width, heads, head dim, q_rank, kv_rank, experts, top, ff of an expert
MIXER_CASES = [(2048, 16, 128, 1024, 512, 16, 2, 1024), (4096, 32, 128, 1536, 512, 32, 4, 1536)]
SFU_TERAOPS = 148 * 16 * 1.965e9 / 1e12            # exponentials, reciprocals: 16 per cycle and SM (nominal)
FP32_TFLOPS = 148 * 128 * 2 * 1.965e9 / 1e12       # FMA pipes at the maximum SM clock (nominal; nothing measures it)


def _measured_hbm() -> float:
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    try:
        with open(path) as f:
            return float(json.load(f)["hbm_gbs"])
    except Exception:
        return 6650.0


def _reporter(args, timer):
    """``report(case, op, fn, ...)``: time ``fn`` and print it beside the slowest of its bounds (HBM bytes, bf16 products, fp32 FMAs,
    special functions)."""
    peak, hbm = _peak_tflops(), _measured_hbm()

    def report(case, op, fn, gbytes=0.0, tflop=0.0, fp32_tflop=0.0, sfu=0.0, like=""):
        if args.only and args.only not in op:
            return
        ms = timer(fn)
        bound = {"hbm": gbytes / hbm * 1e3, "bf16": tflop / peak * 1e3, "fp32": fp32_tflop / FP32_TFLOPS * 1e3, "sfu": sfu / SFU_TERAOPS / 1e9}
        by = max(bound, key=bound.get)
        print(json.dumps(dict(case=case, op=op, us=round(ms * 1e3, 2), bound_us=round(bound[by] * 1e3, 2), bound_by=by,
                              times_bound=round(ms / bound[by], 2), like=like)), flush=True)

    return report


def bench_mixers(args, timer: _Timer) -> None:
    ext = load_ext(required=True)
    report = _reporter(args, _GraphTimer(args.iters, args.warmup, not args.no_flush))
    bf = torch.bfloat16
    mk = lambda *s: (torch.randn(*s, device="cuda") * 0.5).to(bf)                                          # noqa: E731

    for case, (w, h, d, qr, kr, e, top, ff) in enumerate(MIXER_CASES):
        if args.case is not None and args.case != case:
            continue
        # ------------------------------------------------ prompts: 4 x 2048 tokens
        b, s = 4, 2048
        n = b * s
        p = mk(n, 3 * h * d)
        q, f, v = p[:, :h * d], p[:, h * d:2 * h * d], p[:, 2 * h * d:]
        fb, lo, nw = mk(h * d), mk(h * d).abs().clamp(max=0.9), mk(d)
        state = torch.zeros(b, h, d, d, device="cuda")
        report(case, "prompt recurrence", lambda: ext.recurrence(q, f, v, fb, lo, None, state, b, h, d, d),
               gbytes=n * h * d * (3 * 2 + 4) / 1e9, fp32_tflop=6.0 * n * h * d * d / 1e12, like="prompt attention (GPT-J)")
        st1 = torch.zeros(1, h, d, d, device="cuda")
        report(case, "prompt recurrence, 1 x 2048", lambda: ext.recurrence(q[:s], f[:s], v[:s], fb, lo, None, st1, 1, h, d, d),
               gbytes=s * h * d * (3 * 2 + 4) / 1e9, fp32_tflop=6.0 * s * h * d * d / 1e12, like="prompt attention (GPT-J)")
        o = torch.randn(n * h, d, device="cuda")
        report(case, "prompt head norm", lambda: ext.rms_norm(o, nw, 1e-5, 0.0), gbytes=n * h * d * 6 / 1e9, like="layer norm")
        qa, ka, va = (mk(b, s, h, d).permute(0, 2, 1, 3) for _ in range(3))
        fl = 4.0 * b * h * s * s * d * 0.5 / 1e12
        report(case, "prompt attention (GPT-J)", lambda: ext.flash_fwd(qa, ka, va, d ** -0.5, True, 0, None, 1),
               gbytes=4 * n * h * d * 2 / 1e9, tflop=fl)
        oa, lse = ext.flash_fwd(qa, ka, va, d ** -0.5, True, 0, None, 1)
        g, sink = mk(n, h), mk(h)
        report(case, "prompt sink + gate", lambda: ext.sink_gate(oa, lse, sink, g, d), gbytes=n * h * d * 4 / 1e9, like="layer norm")
        x, y, gate, vec = torch.randn(n, w, device="cuda"), mk(n, w), mk(n, w), mk(w)
        report(case, "prompt residual join", lambda: ext.residual_join(x, y, None, None, gate, vec, vec, vec, 1e-5),
               gbytes=n * w * (4 + 2 + 2 + 4 + 2) / 1e9, like="layer norm")
        hb = mk(n, w)
        report(case, "layer norm (GPT-J)", lambda: ext.layernorm_fwd(hb, vec, vec, 1e-5), gbytes=n * w * 4 / 1e9)
        rw, rb = mk(e, w), mk(e)
        up, down = mk(e, ff, w), mk(e, w, ff)
        report(case, "prompt route", lambda: co.moe_route(hb, rw, rb, top), gbytes=n * w * 2 / 1e9, like="layer norm")
        idx, wgt = co.moe_route(hb, rw, rb, top)
        slots, rows, tg, nt = ext.moe_plan(hb, idx, e)
        report(case, "prompt plan + gather", lambda: ext.moe_plan(hb, idx, e), gbytes=n * w * (1 + top) * 2 / 1e9, like="layer norm")
        report(case, "prompt experts up", lambda: ext.moe_grouped(rows, up, tg, nt, 1), tflop=2.0 * n * top * w * ff / 1e12,
               gbytes=(n * top * (w + ff) + e * w * ff) * 2 / 1e9, like="MLP GEMM (GPT-J)")
        a = ext.moe_grouped(rows, up, tg, nt, 1)
        report(case, "prompt experts down", lambda: ext.moe_grouped(a, down, tg, nt, 0), tflop=2.0 * n * top * w * ff / 1e12,
               gbytes=(n * top * (w + ff) + e * w * ff) * 2 / 1e9, like="MLP GEMM (GPT-J)")
        ye = ext.moe_grouped(a, down, tg, nt, 0)
        report(case, "prompt residual join of experts", lambda: ext.residual_join(x, ye, slots, wgt, gate, vec, vec, vec, 1e-5),
               gbytes=n * w * (4 + 2 * top + 2 + 4 + 2) / 1e9, like="layer norm")
        wm = mk(top * ff, w)
        report(case, "MLP GEMM (GPT-J)", lambda: co.gemm(hb, wm), tflop=2.0 * n * w * top * ff / 1e12)
        gu = mk(n, 2 * top * ff)
        report(case, "prompt silu_mul", lambda: ext.silu_mul(gu[:, :top * ff], gu[:, top * ff:]), gbytes=n * top * ff * 6 / 1e9,
               like="layer norm")
        del p, o, qa, ka, va, oa, x, y, gate, hb, rows, a, ye, gu
        # ------------------------------------------------ decode: 1 and 8 rows over 4096 cached tokens
        for rows_n in (1, 8, 64):
            t = 4096
            p = mk(rows_n, 3 * h * d)
            q, f, v = p[:, :h * d], p[:, h * d:2 * h * d], p[:, 2 * h * d:]
            state = torch.zeros(rows_n, h, d, d, device="cuda")
            report(case, f"decode {rows_n} recurrence step", lambda: ext.recurrence_step(q, f, v, fb, lo, nw, None, state, 1e-5, h, d, d),
                   gbytes=rows_n * h * d * d * 8 / 1e9, like="decode attention (GPT-J)")
            cache = mk(rows_n, t, kr)
            lengths = torch.full((rows_n,), t, dtype=torch.int32, device="cuda")
            uk, uv, qd, gd = mk(h * d, kr), mk(h * d, kr), mk(rows_n, h * d), mk(rows_n, h)
            report(case, f"decode {rows_n} latent attention (3 launches)",
                   lambda: ext.latent_decode(qd, uk, uv, cache, lengths, None, sink, gd, d ** -0.5, h),
                   gbytes=(rows_n * t * kr + 2 * h * d * kr) * 2 / 1e9,
                   tflop=4.0 * rows_n * t * h * kr / 1e12, like="decode attention (GPT-J)")
            dq, dkv, wq, wkv = mk(rows_n, qr), mk(rows_n, kr), mk(qr), mk(kr)
            l0 = torch.zeros(rows_n, dtype=torch.int32, device="cuda")
            report(case, f"decode {rows_n} latent norms + append", lambda: ext.latent_prep(dq, wq, dkv, wkv, cache, l0, 1e-5),
                   gbytes=rows_n * (qr + kr) * 4 / 1e9, like="layer norm")
            if rows_n * t * h * d * 4 < 20e9:
                kc, vc = mk(rows_n, h, t, d), mk(rows_n, h, t, d)
                q3 = mk(rows_n, h, d)
                report(case, f"decode {rows_n} attention (GPT-J, 2 launches)", lambda: ext.decode_attn(q3, kc, vc, lengths, d ** -0.5, 0),
                       gbytes=2 * rows_n * t * h * d * 2 / 1e9)
                del kc, vc
            x, y, gate = torch.randn(rows_n, w, device="cuda"), mk(rows_n, w), mk(rows_n, w)
            report(case, f"decode {rows_n} residual join", lambda: ext.residual_join(x, y, None, None, gate, vec, vec, vec, 1e-5),
                   gbytes=rows_n * w * 14 / 1e9, like="layer norm")
            hb = mk(rows_n, w)
            report(case, f"decode {rows_n} layer norm (GPT-J)", lambda: ext.layernorm_fwd(hb, vec, vec, 1e-5), gbytes=rows_n * w * 4 / 1e9)
            report(case, f"decode {rows_n} route", lambda: co.moe_route(hb, rw, rb, top), gbytes=e * w * 2 / 1e9, like="MLP GEMV (GPT-J)")
            idx, wgt = co.moe_route(hb, rw, rb, top)
            used = int(idx.unique().numel())
            report(case, f"decode {rows_n} experts up + down", lambda: co.moe_experts(hb, idx, up, down),
                   gbytes=used * w * ff * 4 / 1e9, like="MLP GEMV (GPT-J)")
            wm, wm2 = mk(top * ff, w), mk(w, top * ff)
            report(case, f"decode {rows_n} MLP GEMV x 2 (GPT-J)", lambda: co.linear(co.linear(hb, wm, None, False, None), wm2, None, False, None),
                   gbytes=2 * w * top * ff * 2 / 1e9)
            del cache


# width, wkv heads x dim, decay rank, inner channels, states, dt_rank, attention heads, kv heads, head dim, linear heads x dim, ff
BRANCH_CASES = [(2048, 32, 64, 64, 4096, 16, 128, 16, 4, 128, 16, 128, 5504), (4096, 64, 64, 128, 8192, 16, 256, 32, 8, 128, 32, 128, 11008)]


def bench_branches(args, timer: _Timer) -> None:
    """The kernels of grouped-query attention, the linear recurrences, the selective scan and the joins (Begovik layers) beside the
    like kernels of the other families."""
    ext = load_ext(required=True)
    report = _reporter(args, _GraphTimer(args.iters, args.warmup, not args.no_flush))
    bf = torch.bfloat16
    mk = lambda *s: (torch.randn(*s, device="cuda") * 0.5).to(bf)                                          # noqa: E731

    for case, (w, rh, rd, rank, inner, ns, dtr, h, g, d, lh, ld, ff) in enumerate(BRANCH_CASES):
        if args.case is not None and args.case != case:
            continue
        vec, nr = mk(w), rh * rd
        w0, u, nw = mk(nr) - 3.0, mk(nr), mk(nr)
        a_log, dtb, dd = mk(inner, ns), mk(inner) - 2.0, mk(inner)
        conv, convb, w_dt = mk(inner, 4), mk(inner), mk(inner, dtr)
        mu, w2 = mk(5, w), mk(nr, rank)
        decay = torch.linspace(0.5, 0.999, lh, device="cuda")
        hw, freq, sink = mk(d), torch.rand(d // 2, device="cuda"), torch.zeros(h, dtype=bf, device="cuda")
        lower = mk(lh * ld).abs().clamp(max=0.9)
        # ------------------------------------------------ prompts: 4 x 2048 and 1 x 2048 tokens
        for b, s in ((4, 2048), (1, 2048)):
            n, tag = b * s, f"prompt {b} x {s} "
            r, k, v, z = mk(n, nr), mk(n, nr), mk(n, nr), torch.randn(n, nr, device="cuda")
            st = torch.zeros(b, rh, rd, rd, device="cuda")
            report(case, tag + "bonus recurrence", lambda: ext.bonus_recurrence(r, k, v, z, w0, u, None, st, b, rh, rd, rd),
                   gbytes=n * nr * 14 / 1e9, fp32_tflop=6.0 * n * nr * rd / 1e12, like="gated recurrence (Moronex)")
            report(case, tag + "gated recurrence, same sizes (Moronex)", lambda: ext.recurrence(r, k, v, w0, w0.sigmoid(), None, st, b, rh, rd, rd),
                   gbytes=n * nr * 10 / 1e9, fp32_tflop=6.0 * n * nr * rd / 1e12)
            q, k, v = mk(n, lh * ld), mk(n, lh * ld), mk(n, lh * ld)
            st2 = torch.zeros(b, lh, ld, ld, device="cuda")
            report(case, tag + "decayed recurrence", lambda: ext.decayed_recurrence(q, k, v, decay, None, st2, b, lh, ld, ld),
                   gbytes=n * lh * ld * 10 / 1e9, fp32_tflop=4.0 * n * lh * ld * ld / 1e12, like="gated recurrence (Moronex)")
            report(case, tag + "gated recurrence (Moronex)", lambda: ext.recurrence(q, k, v, lower, lower, None, st2, b, lh, ld, ld),
                   gbytes=n * lh * ld * 10 / 1e9, fp32_tflop=6.0 * n * lh * ld * ld / 1e12)
            x, zz, dt = mk(n, inner), mk(n, inner), torch.randn(n, inner, device="cuda")
            bc = mk(n, 2 * ns)
            st3 = torch.zeros(b, inner, ns, device="cuda")
            report(case, tag + "selective scan", lambda: ext.selective_scan(x, dt, dtb, a_log, bc[:, :ns], bc[:, ns:], dd, zz, b, None, st3),
                   gbytes=n * inner * 10 / 1e9, fp32_tflop=6.0 * n * inner * ns / 1e12, sfu=1.0 * n * inner * ns, like="gated recurrence (Moronex)")
            qa, ka, va = mk(b, h, s, d), mk(b, g, s, d), mk(b, g, s, d)
            fl = 4.0 * b * h * s * s * d * 0.5 / 1e12
            report(case, tag + "capped attention", lambda: ext.flash_sink_fwd(qa, ka, va, None, sink, None, d ** -0.5, 50.0),
                   gbytes=2 * n * (h + g) * d * 2 / 1e9, tflop=fl, sfu=1.5 * b * h * s * s, like="attention (GPT-J)")
            kf, vf = mk(b, h, s, d), mk(b, h, s, d)
            report(case, tag + "attention (GPT-J)", lambda: ext.flash_fwd(qa, kf, vf, d ** -0.5, True, 0, None, 1),
                   gbytes=4 * n * h * d * 2 / 1e9, tflop=fl)
            del kf, vf
            if b == 1:
                continue
            o, gate = torch.randn(n, nr, device="cuda"), mk(n, nr)
            report(case, tag + "head norm + silu gate", lambda: ext.gated_rms_norm(o, nw, gate, 1e-5, rd, 1), gbytes=n * nr * 8 / 1e9, like="layer norm")
            lw = mk(lh * ld)
            report(case, tag + "norm over heads + sigmoid gate", lambda: ext.gated_rms_norm(o, lw, gate, 1e-5, lh * ld, 0), gbytes=n * nr * 8 / 1e9,
                   like="layer norm")
            hb = mk(n, w)
            report(case, tag + "token shift", lambda: ext.token_shift(hb, mu, b, None, None), gbytes=n * w * 12 / 1e9, like="layer norm")
            report(case, tag + "convolution", lambda: ext.causal_conv(x, conv, convb, b, None, None, True), gbytes=n * inner * 4 / 1e9, like="layer norm")
            p = mk(n, (h + 2 * g) * d)
            kc, vc, l0 = mk(b, g, s, d), mk(b, g, s, d), torch.zeros(b, dtype=torch.int32, device="cuda")
            pos = torch.arange(s, device="cuda")[None].expand(b, s)
            report(case, tag + "norms + rotation + append", lambda: ext.qkv_prep(p[:, :h * d], p[:, h * d:(h + g) * d], p[:, (h + g) * d:], hw, hw, 1e-5,
                                                                              pos, freq, kc, vc, l0), gbytes=n * (h + 2 * g) * d * 4 / 1e9, like="layer norm")
            xs, y1, y2, y3 = torch.randn(n, w, device="cuda"), mk(n, w), mk(n, w), mk(n, w)
            report(case, tag + "join, 2 branches", lambda: co.branch_join(xs, [(y1,), (y2,)], 0.3, 1e-5, [vec, vec]),
                   gbytes=n * w * 16 / 1e9, like="residual join (Moronex)")
            report(case, tag + "join, 3 branches, 2 normed", lambda: co.branch_join(xs, [(y1, vec, 0.5), (y2, vec, 0.5), (y3,)], 0.3, 1e-5, [vec, vec]),
                   gbytes=n * w * 18 / 1e9, like="residual join (Moronex)")
            report(case, tag + "residual join (Moronex)", lambda: ext.residual_join(xs, y1, None, None, y2, vec, vec, vec, 1e-5), gbytes=n * w * 14 / 1e9)
            report(case, tag + "layer norm (GPT-J)", lambda: ext.layernorm_fwd(hb, vec, vec, 1e-5), gbytes=n * w * 4 / 1e9)
            gu = mk(n, 2 * ff)
            report(case, tag + "clamped unit", lambda: ext.clamped_glu(gu[:, :ff], gu[:, ff:], 7.0, 1.702), gbytes=n * ff * 6 / 1e9, like="silu * up (Moronex)")
            report(case, tag + "silu * up (Moronex)", lambda: ext.silu_mul(gu[:, :ff], gu[:, ff:]), gbytes=n * ff * 6 / 1e9)
            wx, wz = mk(dtr + 2 * ns, inner), mk(inner, dtr)
            report(case, tag + "dt product, fp32 result", lambda: co.linear_fp32(x[:, :dtr], wz), gbytes=n * (inner * 4 + dtr * 2) / 1e9,
                   tflop=2.0 * n * inner * dtr / 1e12, like="MLP GEMM (GPT-J)")
            report(case, tag + "x product", lambda: co.linear(x, wx, None, False, None), gbytes=n * inner * 2 / 1e9, tflop=2.0 * n * inner * (dtr + 2 * ns) / 1e12,
                   like="MLP GEMM (GPT-J)")
            ws = mk(4, nr, w)
            xm = mk(4, n, w)
            report(case, tag + "r, k, v, g products", lambda: co.stacked_linear(xm, ws), tflop=8.0 * n * nr * w / 1e12, like="MLP GEMM (GPT-J)")
            wm = mk(4 * w, w)
            report(case, tag + "MLP GEMM (GPT-J)", lambda: co.gemm(hb, wm), tflop=8.0 * n * w * w / 1e12)
            del o, gate, hb, p, xs, y1, y2, y3, gu, xm
        # ------------------------------------------------ decode over 4096 cached tokens
        for n in (1, 8, 64):
            t, tag = 4096, f"decode {n} "
            r, k, v, lo, gate = mk(n, nr), mk(n, nr), mk(n, nr), mk(n, rank), mk(n, nr)
            st = torch.zeros(n, rh, rd, rd, device="cuda")
            report(case, tag + "bonus step", lambda: ext.bonus_step(r, k, v, lo, w2, w0, u, nw, gate, None, st, 1e-5, rh, rd, rd),
                   gbytes=n * nr * rd * 8 / 1e9 + nr * rank * 2 / 1e9, like="recurrence step (Moronex)")
            q, k2, v2 = mk(n, lh * ld), mk(n, lh * ld), mk(n, lh * ld)
            st2 = torch.zeros(n, lh, ld, ld, device="cuda")
            report(case, tag + "decayed step", lambda: ext.decayed_step(q, k2, v2, decay, None, st2, lh, ld, ld), gbytes=n * lh * ld * ld * 8 / 1e9,
                   like="recurrence step (Moronex)")
            nv = mk(ld)
            report(case, tag + "recurrence step (Moronex)", lambda: ext.recurrence_step(q, k2, v2, lower, lower, nv, None, st2, 1e-5, lh, ld, ld),
                   gbytes=n * lh * ld * ld * 8 / 1e9)
            x, zz, dl, bc = mk(n, inner), mk(n, inner), mk(n, dtr), mk(n, 2 * ns)
            st3 = torch.zeros(n, inner, ns, device="cuda")
            report(case, tag + "scan step", lambda: ext.scan_step(x, dl, w_dt, dtb, a_log, bc[:, :ns], bc[:, ns:], dd, zz, None, st3),
                   gbytes=(n * inner * ns * 8 + inner * (dtr + ns) * 2) / 1e9, like="recurrence step (Moronex)")
            cst = torch.zeros(n, 3, inner, device="cuda")
            report(case, tag + "convolution step", lambda: ext.causal_conv(x, conv, convb, n, None, cst, True), gbytes=n * inner * 28 / 1e9, like="layer norm")
            hb, sh = mk(n, w), torch.zeros(n, w, device="cuda")
            report(case, tag + "token shift step", lambda: ext.token_shift(hb, mu, n, None, sh), gbytes=n * w * 20 / 1e9, like="layer norm")
            q3 = mk(n, h, d)
            lengths = torch.full((n,), t, dtype=torch.int32, device="cuda")
            kc, vc = mk(n, g, t, d), mk(n, g, t, d)
            report(case, tag + "capped attention (2 launches)", lambda: ext.grouped_decode(q3, kc, vc, lengths, None, sink, d ** -0.5, 50.0),
                   gbytes=2 * n * t * g * d * 2 / 1e9, like="attention (GPT-J)")
            l1 = torch.full((n,), t - 1, dtype=torch.int32, device="cuda")
            p, pos = mk(n, (h + 2 * g) * d), torch.full((n, 1), t - 1, dtype=torch.long, device="cuda")
            report(case, tag + "norms + rotation + append", lambda: ext.qkv_prep(p[:, :h * d], p[:, h * d:(h + g) * d], p[:, (h + g) * d:], hw, hw, 1e-5, pos,
                                                                              freq, kc, vc, l1), gbytes=n * (h + 2 * g) * d * 4 / 1e9, like="layer norm")
            del kc, vc
            if n * t * h * d * 4 < 20e9:
                kf, vf = mk(n, h, t, d), mk(n, h, t, d)
                report(case, tag + "attention (GPT-J, 2 launches)", lambda: ext.decode_attn(q3, kf, vf, lengths, d ** -0.5, 0), gbytes=2 * n * t * h * d * 2 / 1e9)
                del kf, vf
            xs, y1, y2, y3 = torch.randn(n, w, device="cuda"), mk(n, w), mk(n, w), mk(n, w)
            report(case, tag + "join, 3 branches, 2 normed", lambda: co.branch_join(xs, [(y1, vec, 0.5), (y2, vec, 0.5), (y3,)], 0.3, 1e-5, [vec, vec]),
                   gbytes=n * w * 18 / 1e9, like="layer norm")
            report(case, tag + "layer norm (GPT-J)", lambda: ext.layernorm_fwd(hb, vec, vec, 1e-5), gbytes=n * w * 4 / 1e9)
            ws, xm, wx, wm = mk(4, nr, w), mk(4, n, w), mk(dtr + 2 * ns, inner), mk(4 * w, w)
            report(case, tag + "r, k, v, g products", lambda: co.stacked_linear(xm, ws), gbytes=4 * nr * w * 2 / 1e9, like="MLP GEMV (GPT-J)")
            report(case, tag + "x product", lambda: co.linear(x, wx, None, False, None), gbytes=inner * (dtr + 2 * ns) * 2 / 1e9, like="MLP GEMV (GPT-J)")
            report(case, tag + "MLP GEMV (GPT-J)", lambda: co.linear(hb, wm, None, False, None), gbytes=4 * w * w * 2 / 1e9)
            del ws, wm


# width, streams, attention heads, kv heads, head dim, window, kept, latent dim, rot, vdim, q_rank, kv_rank, memory heads x dim x vdim,
# experts, identity, top, ff
STREAM_CASES = [(2048, 4, 16, 4, 128, 512, 16, 128, 64, 128, 1024, 512, 16, 128, 128, 16, 3, 4, 1344),
                (4096, 4, 32, 8, 128, 1024, 16, 128, 64, 128, 1536, 512, 32, 128, 128, 32, 3, 4, 2688)]


def bench_streams(args, timer: _Timer) -> None:
    """The kernels of the Dekutar layers beside the like kernels of the other families at the same sizes."""
    ext = load_ext(required=True)
    report = _reporter(args, _GraphTimer(args.iters, args.warmup, not args.no_flush))
    bf, none = torch.bfloat16, None
    mk = lambda *s: (torch.randn(*s, device="cuda") * 0.5).to(bf)                                          # noqa: E731
    for case, (w, ns, h, g, d, win, kept, ld, rot, vd, qr, kr, mh, md, mv, e, ident, top, ff) in enumerate(STREAM_CASES):
        if args.case is not None and args.case != case:
            continue
        vec, vq, vk = mk(w), mk(qr), mk(kr)
        w_in, w_out, mix = mk(ns), mk(ns), mk(ns, ns)
        nm, gb, wg = mk(mh * mv), mk(2 * mh), mk(2 * mh, w)
        fb, lo = mk(mh * md), mk(mh * md).abs().clamp(max=0.9)
        decay, sink = torch.linspace(0.5, 0.999, mh, device="cuda"), torch.zeros(h, dtype=bf, device="cuda")
        freq, lfreq = torch.rand(d // 2, device="cuda"), torch.rand(rot // 2, device="cuda")
        rw, rb = mk(e + ident, w) * 0.1, mk(e + ident) * 0.1
        up, down = mk(e, 2 * ff, w), mk(e, w, ff)
        lds = (mv + 4) // 4 * 4
        # ------------------------------------------------ prompts: 4 x 2048 and 1 x 2048 tokens
        for b, s in ((4, 2048), (1, 2048)):
            n, tag = b * s, f"prompt {b} x {s} "
            q, k, v = mk(b, h, s, d), mk(b, g, s, d), mk(b, g, s, d)
            gate, wide = mk(n, h), mk(n, h * vd)
            seen = sum(min(i + 1, win + kept) for i in range(s))
            pairs = b * h * s * s / 2.0
            report(case, tag + "windowed attention + gate", lambda: ext.flash_sink_fwd(q, k, v, none, none, gate, d ** -0.5, 0.0, win, kept),
                   gbytes=2 * n * (h + g) * d * 2 / 1e9, tflop=4.0 * b * h * seen * d / 1e12, sfu=1.0 * b * h * seen, like="attention, window only")
            report(case, tag + "attention, window only", lambda: ext.flash_sink_fwd(q, k, v, none, sink, gate, d ** -0.5, 0.0, win + kept, 0),
                   gbytes=2 * n * (h + g) * d * 2 / 1e9, tflop=4.0 * b * h * seen * d / 1e12, sfu=1.0 * b * h * seen)
            kf, vf = _every_head(k, h // g), _every_head(v, h // g)
            report(case, tag + "attention (GPT-J)", lambda: ext.flash_fwd(q, kf, vf, d ** -0.5, True, 0, none, 1),
                   gbytes=4 * n * h * d * 2 / 1e9, tflop=4.0 * pairs * d / 1e12, sfu=pairs)
            qa, ka, va, kr2 = mk(b, s, h, ld + rot), mk(b, s, h, ld), mk(b, s, h, vd), mk(b, s, kr + rot)
            flat = lambda t: t.permute(0, 2, 1, 3)                                                         # noqa: E731
            report(case, tag + "two-part attention + gate", lambda: ext.flash_sink_fwd(flat(qa)[..., :ld], flat(ka), flat(va), none, none, wide, 0.07, 0.0,
                                                                                       0, 0, none, flat(qa)[..., ld:], kr2[..., kr:]),
                   gbytes=n * (h * (2 * ld + rot + 3 * vd) + rot) * 2 / 1e9, tflop=2.0 * pairs * (ld + rot + vd) / 1e12, sfu=pairs,
                   like="attention with sink + gate (Moronex)")
            report(case, tag + "attention with sink + gate (Moronex)", lambda: ext.flash_sink_fwd(flat(qa)[..., :ld], flat(ka), flat(va), none, sink, gate,
                                                                                                  0.07, 0.0),
                   gbytes=n * h * (2 * ld + 2 * vd) * 2 / 1e9, tflop=2.0 * pairs * (ld + vd) / 1e12, sfu=pairs)
            pm = mk(n, 2 * mh * md + mh * mv)
            mq, mkk, mvv = pm[:, :mh * md], pm[:, mh * md:2 * mh * md], pm[:, 2 * mh * md:]
            z = torch.randn(n, 2 * mh, device="cuda") * 3.0
            st, tp = torch.zeros(b, mh, md, lds, device="cuda"), torch.zeros(b, mh, device="cuda")
            rd, wr, bg, mm = ext.memory_gates(z, gb, 15.0, none, tp, b)
            report(case, tag + "memory gates", lambda: ext.memory_gates(z, gb, 15.0, none, tp, b), gbytes=n * mh * 24 / 1e9, sfu=8.0 * n * mh,
                   like="layer norm")
            report(case, tag + "memory recurrence", lambda: ext.memory_recurrence(mq, mkk, mvv, rd, wr, bg, md ** -0.5, none, st, b, mh, md, mv),
                   gbytes=n * mh * (4 * md + 6 * mv) / 1e9, fp32_tflop=4.0 * n * mh * md * (mv + 1) / 1e12, like="decayed recurrence (Begovik)")
            if md == mv:
                s2 = torch.zeros(b, mh, md, mv, device="cuda")
                report(case, tag + "decayed recurrence (Begovik)", lambda: ext.decayed_recurrence(mq, mkk, mvv, decay, none, s2, b, mh, md, mv),
                       gbytes=n * mh * (4 * md + 6 * mv) / 1e9, fp32_tflop=4.0 * n * mh * md * mv / 1e12)
                report(case, tag + "gated recurrence (Moronex)", lambda: ext.recurrence(mq, mkk, mvv, fb, lo, none, s2, b, mh, md, mv),
                       gbytes=n * mh * (4 * md + 6 * mv) / 1e9, fp32_tflop=6.0 * n * mh * md * mv / 1e12)
            del q, k, v, qa, ka, va, kf, vf
            if b == 1:
                continue
            o, og, nq = torch.randn(n, mh * mv, device="cuda"), mk(n, mh * mv), torch.randn(n, mh, device="cuda")
            report(case, tag + "normaliser + head norm + gate", lambda: ext.gated_rms_norm(o, nm, og, 1e-6, mv, 0, nq, mm), gbytes=n * mh * mv * 8 / 1e9,
                   like="head norm + gate (Begovik)")
            report(case, tag + "head norm + gate (Begovik)", lambda: ext.gated_rms_norm(o, nm, og, 1e-6, mv, 0), gbytes=n * mh * mv * 8 / 1e9)
            hb = mk(n, w)
            report(case, tag + "gate logits, fp32 result", lambda: co.linear_fp32(hb, wg), gbytes=n * w * 2 / 1e9, like="route (Moronex)")
            pos, l0 = torch.arange(s, device="cuda")[None].expand(b, s), torch.zeros(b, dtype=torch.int32, device="cuda")
            pa = mk(n, (h + g) * d)
            kc, vc = mk(b, g, s, d), mk(b, g, s, d)
            report(case, tag + "norms + rotation + append", lambda: ext.qkv_prep(pa[:, :h * d], pa[:, h * d:], pa[:, h * d:], none, none, 1e-6, pos, freq, kc,
                                                                              vc, l0), gbytes=n * (2 * h + 3 * g) * d * 2 / 1e9, like="layer norm")
            pl, lc = mk(n, qr + kr + rot), mk(b, s, kr + rot)
            report(case, tag + "latent norms + rotation + append", lambda: ext.latent_prep(pl[:, :qr], vq, pl[:, qr:], vk, lc, l0, 1e-6, pos, lfreq, True),
                   gbytes=n * (2 * qr + 3 * kr + 2 * rot) * 2 / 1e9, like="layer norm")
            ql = mk(b, s, h, ld + rot)
            report(case, tag + "query rotation in place", lambda: ext.rotate_halves_(ql, pos, lfreq), gbytes=n * h * rot * 4 / 1e9, like="layer norm")
            x, y, sh, sg = torch.randn(n, ns, w, device="cuda"), mk(n, w), mk(n, w), mk(n, 8)[:, :1]
            report(case, tag + f"join of {ns} streams", lambda: ext.hyper_join(x, y, none, none, none, 0, none, none, none, w_out, mix, w_in, vec, 1e-6, 1.0),
                   gbytes=n * w * (8 * ns + 4) / 1e9, like="residual join (Moronex)")
            x1, gt = torch.randn(n, w, device="cuda"), mk(n, w)
            report(case, tag + "residual join (Moronex)", lambda: ext.residual_join(x1, y, none, none, gt, vec, vec, vec, 1e-5), gbytes=n * w * 14 / 1e9)
            report(case, tag + "layer norm (GPT-J)", lambda: ext.layernorm_fwd(hb, vec, vec, 1e-5), gbytes=n * w * 4 / 1e9)
            report(case, tag + "route, scored", lambda: co.moe_route(hb, rw, rb, top, True), gbytes=n * w * 2 / 1e9, like="route (Moronex)")
            report(case, tag + "route (Moronex)", lambda: co.moe_route(hb, rw, rb, top), gbytes=n * w * 2 / 1e9)
            idx, wgt = co.moe_route(hb, rw, rb, top, True)
            real = int((idx < e).sum())
            slots, rows, tg, nt = ext.moe_plan(hb, idx, e)
            report(case, tag + "plan + gather", lambda: ext.moe_plan(hb, idx, e), gbytes=(n + real) * w * 2 / 1e9, like="layer norm")
            report(case, tag + "gated experts up", lambda: ext.moe_grouped(rows, up, tg, nt, 2), tflop=4.0 * real * w * ff / 1e12,
                   gbytes=(real * (w + ff) + 2 * e * w * ff) * 2 / 1e9, like="experts up, relu^2 (Moronex)")
            report(case, tag + "experts up, relu^2 (Moronex)", lambda: ext.moe_grouped(rows, up, tg, nt, 1), tflop=4.0 * real * w * ff / 1e12,
                   gbytes=(real * (w + 2 * ff) + 2 * e * w * ff) * 2 / 1e9)
            a = ext.moe_grouped(rows, up, tg, nt, 2)
            report(case, tag + "experts down", lambda: ext.moe_grouped(a, down, tg, nt, 0), tflop=2.0 * real * w * ff / 1e12,
                   gbytes=(real * (w + ff) + e * w * ff) * 2 / 1e9, like="experts up, relu^2 (Moronex)")
            ye = ext.moe_grouped(a, down, tg, nt, 0)
            report(case, tag + f"join of {ns} streams, experts + shared",
                   lambda: ext.hyper_join(x, ye, slots, wgt, idx, e, hb, sh, sg, w_out, mix, w_in, vec, 1e-6, 1.0),
                   gbytes=(n * w * (8 * ns + 4) + (real + n) * w * 2) / 1e9, like="residual join of experts (Moronex)")
            report(case, tag + "residual join of experts (Moronex)", lambda: ext.residual_join(x1, ye, slots.clamp(min=0), wgt, gt, vec, vec, vec, 1e-5),
                   gbytes=n * w * (12 + 2 * top) / 1e9)
            del o, og, hb, pa, x, y, sh, rows, a, ye, x1, gt
        # ------------------------------------------------ decode over 4096 cached tokens
        for n in (1, 8, 64):
            t, tag = 4096, f"decode {n} "
            lengths = torch.full((n,), t, dtype=torch.int32, device="cuda")
            l1, pos = lengths - 1, torch.full((n, 1), t - 1, dtype=torch.long, device="cuda")
            q3, gate, kc, vc = mk(n, h, d), mk(n, h), mk(n, g, t, d), mk(n, g, t, d)
            report(case, tag + "windowed attention + gate (2 launches)", lambda: ext.grouped_decode(q3, kc, vc, lengths, none, none, d ** -0.5, 0.0, gate, win, kept),
                   gbytes=2 * n * (win + kept) * g * d * 2 / 1e9, like="attention over as many keys (Begovik)")
            ks, vs, ls = mk(n, g, win + kept, d), mk(n, g, win + kept, d), torch.full((n,), win + kept, dtype=torch.int32, device="cuda")
            report(case, tag + "attention over as many keys (Begovik)", lambda: ext.grouped_decode(q3, ks, vs, ls, none, sink, d ** -0.5, 0.0),
                   gbytes=2 * n * (win + kept) * g * d * 2 / 1e9)
            pa = mk(n, (h + g) * d)
            report(case, tag + "norms + rotation + append", lambda: ext.qkv_prep(pa[:, :h * d], pa[:, h * d:], pa[:, h * d:], none, none, 1e-6, pos, freq, kc,
                                                                              vc, l1), gbytes=n * (2 * h + 3 * g) * d * 2 / 1e9, like="layer norm")
            del kc, vc, ks, vs
            uk, uv, ql, wide, lc = mk(h * ld, kr), mk(h * vd, kr), mk(n, h * (ld + rot)), mk(n, h * vd), mk(n, t, kr + rot)
            report(case, tag + "rotated latent attention (3 launches)",
                   lambda: ext.latent_decode(ql, uk, uv, lc, lengths, none, none, wide, 0.07, h, pos, lfreq),
                   gbytes=(n * t * (kr + rot) + h * (ld + vd) * kr) * 2 / 1e9, tflop=2.0 * n * t * h * (2 * kr + rot) / 1e12, like="latent attention (Moronex)")
            lm, qm = mk(n, t, kr), mk(n, h * ld)
            report(case, tag + "latent attention (Moronex)", lambda: ext.latent_decode(qm, uk, uv, lm, lengths, none, sink, gate, 0.07, h),
                   gbytes=(n * t * kr + h * (ld + vd) * kr) * 2 / 1e9, tflop=4.0 * n * t * h * kr / 1e12)
            pl = mk(n, qr + kr + rot)
            report(case, tag + "latent norms + rotation + append", lambda: ext.latent_prep(pl[:, :qr], vq, pl[:, qr:], vk, lc, l1, 1e-6, pos, lfreq),
                   gbytes=n * (qr + kr + rot) * 4 / 1e9, like="layer norm")
            del lc, lm
            mq, mkk, mvv, og, hb = mk(n, mh * md), mk(n, mh * md), mk(n, mh * mv), mk(n, mh * mv), mk(n, w)
            st, tp = torch.zeros(n, mh, md, lds, device="cuda"), torch.zeros(n, mh, device="cuda")
            report(case, tag + "memory step", lambda: ext.memory_step(mq, mkk, mvv, hb, wg, gb, 15.0, og, nm, none, st, tp, md ** -0.5, 1e-6, mh, md, mv),
                   gbytes=(n * mh * md * (mv + 1) * 8 + 2 * mh * w * 2) / 1e9, like="recurrence step (Moronex)")
            if md == mv:
                s2, nv = torch.zeros(n, mh, md, mv, device="cuda"), mk(mv)
                report(case, tag + "recurrence step (Moronex)", lambda: ext.recurrence_step(mq, mkk, mvv, fb, lo, nv, none, s2, 1e-5, mh, md, mv),
                       gbytes=n * mh * md * mv * 8 / 1e9)
            x, y, sh, sg = torch.randn(n, ns, w, device="cuda"), mk(n, w), mk(n, w), mk(n, 8)[:, :1]
            report(case, tag + f"join of {ns} streams", lambda: ext.hyper_join(x, y, none, none, none, 0, none, none, none, w_out, mix, w_in, vec, 1e-6, 1.0),
                   gbytes=n * w * (8 * ns + 4) / 1e9, like="residual join (Moronex)")
            x1, gt = torch.randn(n, w, device="cuda"), mk(n, w)
            report(case, tag + "residual join (Moronex)", lambda: ext.residual_join(x1, y, none, none, gt, vec, vec, vec, 1e-5), gbytes=n * w * 14 / 1e9)
            report(case, tag + "layer norm (GPT-J)", lambda: ext.layernorm_fwd(hb, vec, vec, 1e-5), gbytes=n * w * 4 / 1e9)
            report(case, tag + "route, scored", lambda: co.moe_route(hb, rw, rb, top, True), gbytes=(e + ident) * w * 2 / 1e9, like="route (Moronex)")
            report(case, tag + "route (Moronex)", lambda: co.moe_route(hb, rw, rb, top), gbytes=(e + ident) * w * 2 / 1e9)
            idx, wgt = co.moe_route(hb, rw, rb, top, True)
            used = int(idx[idx < e].unique().numel())
            report(case, tag + "gated experts up + down", lambda: co.moe_experts(hb, idx, up, down, "silu"), gbytes=used * w * ff * 6 / 1e9,
                   like="experts up + down, relu^2 (Moronex)")
            up1 = mk(e, ff, w)
            report(case, tag + "experts up + down, relu^2 (Moronex)", lambda: co.moe_experts(hb, idx, up1, down), gbytes=used * w * ff * 4 / 1e9)
            ye, slots = co.moe_experts(hb, idx, up, down, "silu")
            report(case, tag + f"join of {ns} streams, experts + shared",
                   lambda: ext.hyper_join(x, ye, slots, wgt, idx, e, hb, sh, sg, w_out, mix, w_in, vec, 1e-6, 1.0),
                   gbytes=n * w * (8 * ns + 6 + 2 * top) / 1e9, like="residual join (Moronex)")
            del up1


# width, heads, kv heads, head dim, experts, top, ff of an expert, token dim, taps
TALK_CASES = [(2048, 16, 4, 128, 16, 3, 1344, 256, 4), (4096, 32, 8, 128, 32, 3, 2688, 256, 4), (4096, 32, 4, 128, 32, 3, 2688, 256, 4)]


def bench_talk(args, timer: _Timer) -> None:
    """The kernels of the Masezen layers beside the like kernels of the other families at the same sizes."""
    ext = load_ext(required=True)
    report = _reporter(args, _GraphTimer(args.iters, args.warmup, not args.no_flush))
    bf, none = torch.bfloat16, None
    mk = lambda *s: (torch.randn(*s, device="cuda") * 0.5).to(bf)                                          # noqa: E731
    for case, (w, h, g, d, e, top, ff, td, taps) in enumerate(TALK_CASES):
        if args.case is not None and args.case != case:
            continue
        vec, vd, talk, conv, one = mk(w), mk(d), mk(h, h), mk(w, taps), mk(1)
        sink, freq = torch.zeros(h, dtype=bf, device="cuda"), torch.rand(d // 2, device="cuda")
        rw, rb = mk(e, w) * 0.1, mk(e) * 0.1
        up, down, dense, wg, wp, table = mk(e, 2 * ff, w), mk(e, w, ff), mk(4 * w, w), mk(td, w), mk(w, td), mk(50400, 8 * td)
        clamped = lambda rows, tg, nt: ext.moe_grouped(rows, up, tg, nt, 3, 7.0, 1.702)                    # noqa: E731
        # ------------------------------------------------ prompts: 4 x 2048 and 1 x 2048 tokens
        for b, s in ((4, 2048), (1, 2048)):
            n, tag = b * s, f"prompt {b} x {s} "
            q, k, v, gate = mk(b, s, h, g * d), mk(b, 1, s, g * d), mk(b, s, g, d), mk(n, h * d)
            flat = lambda t: t.permute(0, 2, 1, 3)                                                         # noqa: E731
            pairs = b * h * s * s / 2.0
            report(case, tag + "attention, mixed heads + gate", lambda: ext.flash_wide_fwd(flat(q), k, flat(v), none, none, gate, d ** -0.5),
                   gbytes=n * (3 * h + 2 * g) * d * 2 / 1e9, tflop=2.0 * pairs * (2 * d + h) / 1e12, sfu=pairs, like="attention, heads alone (Begovik)")
            qg, kg = mk(b, s, h, d), mk(b, s, g, d)
            report(case, tag + "attention, heads alone (Begovik)", lambda: ext.flash_sink_fwd(flat(qg), flat(kg), flat(v), none, sink, none, d ** -0.5, 0.0),
                   gbytes=n * (2 * h + 2 * g) * d * 2 / 1e9, tflop=4.0 * pairs * d / 1e12, sfu=pairs)
            pos, l0 = torch.arange(s, device="cuda")[None].expand(b, s), torch.zeros(b, dtype=torch.int32, device="cuda")
            pa = mk(n, (h + g) * d)
            ks, vs = mk(b, s, g, d), mk(b, s, g, d)
            report(case, tag + "norms + rotation + mix + append",
                   lambda: ext.head_prep(pa[:, :h * d], pa[:, h * d:], pa[:, h * d:], vd, vd, 1e-6, pos, freq, True, 1.1, talk, flat(ks), flat(vs), l0),
                   gbytes=n * (h + h * g + 3 * g) * d * 2 / 1e9, fp32_tflop=2.0 * n * h * h * d / 1e12, like="norms + rotation + append (Begovik)")
            kc, vc = mk(b, g, s, d), mk(b, g, s, d)
            report(case, tag + "norms + rotation by halves + append",
                   lambda: ext.head_prep(pa[:, :h * d], pa[:, h * d:], pa[:, h * d:], vd, vd, 1e-6, pos, freq, True, 1.1, none, kc, vc, l0),
                   gbytes=n * (2 * h + 3 * g) * d * 2 / 1e9, like="norms + rotation + append (Begovik)")
            report(case, tag + "norms + rotation + append (Begovik)",
                   lambda: ext.qkv_prep(pa[:, :h * d], pa[:, h * d:], pa[:, h * d:], vd, vd, 1e-6, pos, freq, kc, vc, l0),
                   gbytes=n * (2 * h + 3 * g) * d * 2 / 1e9, like="layer norm")
            del q, k, v, qg, kg, pa, ks, vs, kc, vc
            hb, x, y, sh = mk(n, w), torch.randn(n, w, device="cuda"), mk(n, w), mk(n, w)
            report(case, tag + "input convolution", lambda: ext.causal_conv(hb, conv, none, b, none, none, False, True), gbytes=n * w * 4 / 1e9,
                   like="layer norm (GPT-J)")
            report(case, tag + "join of mixer + dense, copy", lambda: co.branch_join(x, [(y, vec, 1.0, False), (sh, vec, 1.0, False)], 1.0, 1e-6, [], bf),
                   gbytes=n * w * 14 / 1e9, like="residual join (Moronex)")
            report(case, tag + "join of token input + norm", lambda: co.branch_join(x, [(y, vec)], 1.0, 1e-6, [one]), gbytes=n * w * 12 / 1e9,
                   like="residual join (Moronex)")
            report(case, tag + "residual join (Moronex)", lambda: ext.residual_join(x, y, none, none, sh, vec, vec, vec, 1e-5), gbytes=n * w * 14 / 1e9)
            report(case, tag + "layer norm (GPT-J)", lambda: ext.layernorm_fwd(hb, vec, vec, 1e-5), gbytes=n * w * 4 / 1e9)
            z, ids = mk(n, td), torch.randint(0, 50400, (n,), device="cuda")
            report(case, tag + "token input: gate product", lambda: co.linear(hb, wg, none, False, none), gbytes=n * (w + td) * 2 / 1e9,
                   tflop=2.0 * n * w * td / 1e12, like="MLP GEMM (GPT-J)")
            report(case, tag + "token input: gelu * entry", lambda: ext.token_gate(z, ids, table, td), gbytes=n * td * 6 / 1e9, like="layer norm (GPT-J)")
            report(case, tag + "token input: product", lambda: co.linear(z, wp, none, False, none), gbytes=n * (w + td) * 2 / 1e9,
                   tflop=2.0 * n * w * td / 1e12, like="MLP GEMM (GPT-J)")
            report(case, tag + "dense up, relu^2", lambda: co.linear(hb, dense, none, False, "relu2"), tflop=8.0 * n * w * w / 1e12, like="MLP GEMM (GPT-J)")
            report(case, tag + "MLP GEMM (GPT-J)", lambda: co.linear(hb, dense, none, False, "gelu_new"), tflop=8.0 * n * w * w / 1e12)
            report(case, tag + "route, sigmoid", lambda: co.moe_route(hb, rw, none, top, "sigmoid"), gbytes=n * w * 2 / 1e9, like="route (Moronex)")
            report(case, tag + "route (Moronex)", lambda: co.moe_route(hb, rw, rb, top), gbytes=n * w * 2 / 1e9)
            idx, wgt = co.moe_route(hb, rw, none, top, "sigmoid")
            real = n * top
            slots, rows, tg, nt = ext.moe_plan(hb, idx, e, wgt)
            report(case, tag + "plan + scaled gather", lambda: ext.moe_plan(hb, idx, e, wgt), gbytes=(n + real) * w * 2 / 1e9, like="plan + gather (Moronex)")
            report(case, tag + "plan + gather (Moronex)", lambda: ext.moe_plan(hb, idx, e), gbytes=(n + real) * w * 2 / 1e9)
            report(case, tag + "clamped experts up", lambda: clamped(rows, tg, nt), tflop=4.0 * real * w * ff / 1e12,
                   gbytes=(real * (w + ff) + 2 * e * w * ff) * 2 / 1e9, like="gated experts up (Dekutar)")
            report(case, tag + "gated experts up (Dekutar)", lambda: ext.moe_grouped(rows, up, tg, nt, 2), tflop=4.0 * real * w * ff / 1e12,
                   gbytes=(real * (w + ff) + 2 * e * w * ff) * 2 / 1e9)
            a = clamped(rows, tg, nt)
            ye = ext.moe_grouped(a, down, tg, nt, 0)
            report(case, tag + "join of mixer + experts + shared, copy",
                   lambda: co.branch_join(x, [(y, vec, 1.0, False), (ye, vec, 1.0, False, slots, top), (sh, vec, 1.0, False)], 1.0, 1e-6, [], bf),
                   gbytes=n * w * (14 + 2 * top) / 1e9, like="residual join of experts (Moronex)")
            report(case, tag + "residual join of experts (Moronex)", lambda: ext.residual_join(x, ye, slots, wgt, sh, vec, vec, vec, 1e-5),
                   gbytes=n * w * (12 + 2 * top) / 1e9)
            del hb, x, y, sh, rows, a, ye
        # ------------------------------------------------ decode over 4096 cached tokens
        for n in (1, 8, 64):
            t, tag = 4096, f"decode {n} "
            lengths = torch.full((n,), t, dtype=torch.int32, device="cuda")
            l1, pos = lengths - 1, torch.full((n, 1), t - 1, dtype=torch.long, device="cuda")
            q, gate, ks, vs = mk(n, h, g * d), mk(n, h * d), mk(n, 1, t, g * d), mk(n, 1, t, g * d)
            report(case, tag + "attention, mixed heads + gate (2 launches)",
                   lambda: ext.grouped_decode(q, ks, vs, lengths, none, none, d ** -0.5, 0.0, gate, 0, 0, none, g),
                   gbytes=2 * n * t * g * d * 2 / 1e9, like="attention, heads alone (Begovik, 2 launches)")
            pa = mk(n, (h + g) * d)
            heads = lambda c: c.view(n, t, g, d).transpose(1, 2)                                           # noqa: E731
            report(case, tag + "norms + rotation + mix + append",
                   lambda: ext.head_prep(pa[:, :h * d], pa[:, h * d:], pa[:, h * d:], vd, vd, 1e-6, pos, freq, True, 1.1, talk, heads(ks), heads(vs), l1),
                   gbytes=n * (h + h * g + 3 * g) * d * 2 / 1e9, like="norms + rotation + append (Begovik)")
            q3, kc, vc = mk(n, h, d), ks.view(n, g, t, d), vs.view(n, g, t, d)
            report(case, tag + "attention, heads alone (Begovik, 2 launches)", lambda: ext.grouped_decode(q3, kc, vc, lengths, none, sink, d ** -0.5, 0.0),
                   gbytes=2 * n * t * g * d * 2 / 1e9)
            report(case, tag + "norms + rotation + append (Begovik)",
                   lambda: ext.qkv_prep(pa[:, :h * d], pa[:, h * d:], pa[:, h * d:], vd, vd, 1e-6, pos, freq, kc, vc, l1),
                   gbytes=n * (2 * h + 3 * g) * d * 2 / 1e9)
            del ks, vs, kc, vc
            hb, x, y, sh, state = mk(n, w), torch.randn(n, w, device="cuda"), mk(n, w), mk(n, w), torch.zeros(n, taps - 1, w, device="cuda")
            report(case, tag + "join of token input + norm + convolution", lambda: co.branch_join(x, [(y, vec)], 1.0, 1e-6, [one], none, (conv, state, none)),
                   gbytes=n * w * (14 + 8 * (taps - 1)) / 1e9, like="residual join (Moronex)")
            report(case, tag + "residual join (Moronex)", lambda: ext.residual_join(x, y, none, none, sh, vec, vec, vec, 1e-5), gbytes=n * w * 14 / 1e9)
            z, ids = mk(n, td), torch.randint(0, 50400, (n,), device="cuda")
            report(case, tag + "token input (3 launches)", lambda: co.linear(ext.token_gate(co.linear(hb, wg, none, False, none), ids, table, td), wp, none, False, none),
                   gbytes=2 * w * td * 2 / 1e9, like="route (Moronex)")
            report(case, tag + "dense up, relu^2", lambda: co.linear(hb, dense, none, False, "relu2"), gbytes=8 * w * w / 1e9, like="MLP GEMV (GPT-J)")
            report(case, tag + "MLP GEMV (GPT-J)", lambda: co.linear(hb, dense, none, False, "gelu_new"), gbytes=8 * w * w / 1e9)
            report(case, tag + "route, sigmoid", lambda: co.moe_route(hb, rw, none, top, "sigmoid"), gbytes=e * w * 2 / 1e9, like="route (Moronex)")
            report(case, tag + "route (Moronex)", lambda: co.moe_route(hb, rw, rb, top), gbytes=e * w * 2 / 1e9)
            idx, wgt = co.moe_route(hb, rw, none, top, "sigmoid")
            used = int(idx.unique().numel())
            report(case, tag + "clamped experts up + down", lambda: co.moe_experts(hb, idx, up, down, "clamped", 7.0, 1.702, wgt), gbytes=used * w * ff * 6 / 1e9,
                   like="gated experts up + down (Dekutar)")
            report(case, tag + "gated experts up + down (Dekutar)", lambda: co.moe_experts(hb, idx, up, down, "silu"), gbytes=used * w * ff * 6 / 1e9)
            ye, slots = co.moe_experts(hb, idx, up, down, "clamped", 7.0, 1.702, wgt)
            report(case, tag + "join of mixer + experts + shared, copy",
                   lambda: co.branch_join(x, [(y, vec, 1.0, False), (ye, vec, 1.0, False, slots, top), (sh, vec, 1.0, False)], 1.0, 1e-6, [], bf),
                   gbytes=n * w * (14 + 2 * top) / 1e9, like="residual join (Moronex)")


def _every_head(t: torch.Tensor, per: int) -> torch.Tensor:
    """Every key / value head ``per`` times: what attention without groups reads."""
    b, g, s, d = t.shape
    return t[:, :, None].expand(b, g, per, s, d).reshape(b, g * per, s, d)


def main() -> None:
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--op", choices=["gemm", "attention", "mixers", "branches", "streams", "talk"], required=True)
    ap.add_argument("--case", type=int, default=None, help="index into the op's shape list")
    ap.add_argument("--iters", type=int, default=20)
    ap.add_argument("--warmup", type=int, default=5)
    ap.add_argument("--causal", type=int, default=None, help="attention: 1 / 0 to run only one mask")
    ap.add_argument("--no-baseline", action="store_true", help="skip the library / legacy-kernel baseline")
    ap.add_argument("--no-flush", action="store_true", help="do not write a 256 MB buffer between timed calls")
    ap.add_argument("--only", default="", help="mixers, branches, streams, talk: only the entries whose name contains this")
    args = ap.parse_args()
    timer = _Timer(args.iters, args.warmup, not args.no_flush)
    with torch.no_grad():
        {"gemm": bench_gemm, "attention": bench_attention, "mixers": bench_mixers, "branches": bench_branches, "streams": bench_streams,
         "talk": bench_talk}[args.op](args, timer)


if __name__ == "__main__":
    main()
