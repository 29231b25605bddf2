"""The kernels behind Moronex against the fp32 PyTorch statements of the same ops, over sizes that do and do not fit the
vector widths and tiles, and the whole model on the GPU against the plain implementation in ``plain_moronex.py``."""
import pytest
import torch

import oslo_b200 as ob
from oslo_b200 import ops
from oslo_b200.ops import reference as ref

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16, torch.float16]
TOL = {torch.float32: 2e-5, torch.bfloat16: 2e-2, torch.float16: 3e-3}


def rnd(*shape, dtype=torch.float32, scale=1.0, seed=0):
    g = torch.Generator().manual_seed(seed + 7919 * len(shape) + sum(shape))
    return (torch.randn(*shape, generator=g) * scale).to(dtype).cuda()


def close(got, want, dtype, factor=1.0):
    got, want = got.float(), want.float()
    assert got.shape == want.shape
    assert torch.isfinite(got).all()
    scale = want.abs().amax().clamp(min=1e-3)
    err = ((got - want).abs().amax() / scale).item()
    assert err < factor * TOL[dtype], err


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,cols", [(1, 256), (3, 40), (130, 96), (70, 33), (5, 1030), (65, 4096)])
def test_rms_norm(dtype, rows, cols):
    wide = rnd(rows, cols + 8, dtype=dtype)
    for x in (wide[:, :cols], wide[:, 4:4 + cols].float(), wide[:, 3:3 + cols]):
        w = rnd(cols, dtype=dtype, scale=0.3)
        for offset in (0.0, 1.0):
            close(ops.rms_norm(x, w, 1e-3, offset), ref.rms_norm(x, w, 1e-3, offset), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,cols,top", [(1, 256, 0), (7, 100, 0), (33, 1024, 2), (5, 37, 3), (129, 512, 1)])
@pytest.mark.parametrize("nxt", [True, False])
def test_residual_join(dtype, rows, cols, top, nxt):
    x, gate = rnd(rows, cols), rnd(rows, cols + 16, dtype=dtype, seed=2)[:, 8:8 + cols]
    b, wp, wn = rnd(cols, dtype=dtype, seed=3), rnd(cols, dtype=dtype, scale=0.2, seed=4), rnd(cols, dtype=dtype, scale=0.2, seed=5)
    wn = wn if nxt else None
    if top == 0:
        cases = [(rnd(rows, cols, dtype=dtype, seed=6), None, None)]
    else:
        sw = torch.softmax(rnd(rows, top, seed=8), -1)
        slots = torch.randperm(rows * top + 5, device="cuda")[:rows * top].view(rows, top).to(torch.int32)
        cases = [(rnd(rows * top, cols, dtype=dtype, seed=6), None, sw), (rnd(rows * top + 5, cols, dtype=dtype, seed=7), slots, sw)]
    for y, slots, sw in cases:
        x1, h1 = ops.residual_join(x, y, gate, b, wp, wn, 1e-4, slots, sw)
        x2, h2 = ref.residual_join(x, y, gate, b, wp, wn, 1e-4, slots, sw)
        assert x1.dtype == torch.float32
        close(x1, x2, torch.float32)                  # the stream is 32-bit whatever the storage type
        assert (h1 is None) == (not nxt)
        if nxt:
            close(h1, h2, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cols", [96, 50, 2048])
def test_silu_mul(dtype, cols):
    t = rnd(9, 2 * cols + 8, dtype=dtype)
    close(ops.silu_mul(t[:, :cols], t[:, cols:2 * cols]), ref.silu_mul(t[:, :cols], t[:, cols:2 * cols]), dtype)


def recurrence_inputs(batch, s, heads, dim, vdim, dtype, seed=0):
    n = batch * s
    total = 2 * heads * dim + heads * vdim
    p = rnd(n, total + 8, dtype=dtype, seed=seed)
    q, f, v = p[:, :heads * dim], p[:, heads * dim:2 * heads * dim], p[:, 2 * heads * dim:total]
    fb = rnd(heads * dim, dtype=dtype, seed=seed + 1) + 2.0
    lower = torch.rand(heads * dim, generator=torch.Generator().manual_seed(seed)).mul(0.9).to(dtype).cuda()
    return q, f, v, fb.to(dtype), lower


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("batch,s,heads,dim,vdim", [(2, 37, 3, 48, 64), (1, 1, 2, 16, 8), (1, 200, 1, 12, 20), (2, 17, 2, 100, 33),
                                                    (1, 150, 2, 128, 128), (3, 5, 1, 256, 24), (1, 9, 1, 300, 40), (2, 64, 2, 30, 72)])
def test_recurrence(dtype, batch, s, heads, dim, vdim):
    q, f, v, fb, lower = recurrence_inputs(batch, s, heads, dim, vdim, dtype)
    ext = ops.load_ext(required=True)
    s0 = rnd(batch, heads, dim, vdim, scale=0.5)
    keep = (torch.rand(batch, s + 3, device="cuda") > 0.25).to(torch.uint8)[:, 3:]
    for kp in (None, keep):
        for start in (None, s0):
            want, end = ref.recurrence(q, f, v, fb, lower, kp, start, batch, heads, dim, vdim)
            for chunks in (0, 1, 2, 5):
                st = start.clone() if start is not None else torch.zeros_like(s0)
                got = ext.recurrence(q, f, v, fb, lower, kp, st, batch, heads, dim, vdim, chunks)
                close(got, want, torch.float32)
                close(st, end, torch.float32)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("batch,heads,dim,vdim", [(1, 4, 48, 64), (5, 3, 20, 30), (2, 16, 128, 128), (70, 2, 64, 256), (1, 1, 7, 2100)])
def test_recurrence_step_is_one_token_of_the_recurrence(dtype, batch, heads, dim, vdim):
    q, f, v, fb, lower = recurrence_inputs(batch, 1, heads, dim, vdim, dtype)
    w = rnd(vdim, dtype=dtype)
    s0 = rnd(batch, heads, dim, vdim)
    for keep in (None, (torch.arange(batch, device="cuda") % 2 == 0).to(torch.uint8)[:, None]):
        want, end = ref.recurrence(q, f, v, fb, lower, keep, s0, batch, heads, dim, vdim)
        st = s0.clone()
        got = ops.gated_recurrence(q, f, v, fb, lower, w, 1e-5, batch, heads, keep, st)
        close(got, ref.rms_norm(want, w, 1e-5).view(batch, -1), dtype)
        close(st, end, torch.float32)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("batch,sq,sk,heads,dim,vdim", [(2, 50, 50, 3, 64, 64), (1, 1, 9, 2, 20, 12), (2, 33, 70, 2, 48, 80),
                                                        (1, 140, 300, 2, 128, 128), (1, 19, 19, 1, 300, 20), (2, 130, 130, 2, 192, 128)])
def test_sink_attention(dtype, batch, sq, sk, heads, dim, vdim):
    q, k, v = (rnd(batch, n, heads, d, dtype=dtype, seed=i) for i, (n, d) in enumerate(((sq, dim), (sk, dim), (sk, vdim))))
    sink, gate = rnd(heads, dtype=dtype, scale=2.0), rnd(batch * sq, heads + 8, dtype=dtype)[:, :heads]
    keep = torch.ones(batch, sk, dtype=torch.uint8, device="cuda")
    keep[0, :min(7, sk - 1)] = 0
    for kp in (None, keep):
        want, _ = ref.sink_attention(q, k, v, kp, sink, gate, dim ** -0.5)
        close(ops.sink_attention(q, k, v, kp, sink, gate, dim ** -0.5), want, dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("batch,heads,dim,vdim,rank,tmax,length", [(2, 4, 64, 64, 96, 200, 131), (1, 3, 20, 12, 40, 64, 1),
                                                                   (3, 17, 48, 80, 100, 96, 96), (1, 16, 128, 128, 512, 1500, 1400),
                                                                   (2, 8, 32, 64, 1000, 300, 290), (9, 2, 16, 24, 64, 33, 20),
                                                                   (1, 40, 64, 64, 256, 700, 641), (2, 5, 64, 64, 320, 400, 390)])
def test_latent_decode(dtype, batch, heads, dim, vdim, rank, tmax, length):
    q = rnd(batch, heads * dim, dtype=dtype)
    uk, uv = rnd(heads * dim, rank, dtype=dtype, scale=rank ** -0.5), rnd(heads * vdim, rank, dtype=dtype, scale=rank ** -0.5, seed=3)
    cache = rnd(batch, tmax, rank, dtype=dtype)
    cache[:, length:] = float("nan")                      # nothing beyond the valid length may be touched
    lengths = torch.full((batch,), length, dtype=torch.int32, device="cuda")
    sink, gate = rnd(heads, dtype=dtype, scale=2.0), rnd(batch, heads + 8, dtype=dtype)[:, :heads]
    keep = torch.ones(batch, length, dtype=torch.uint8, device="cuda")
    keep[-1, :min(5, length - 1)] = 0
    clean = torch.nan_to_num(cache)
    for kp in (None, keep):
        want = ref.latent_decode(q, uk, uv, clean, lengths, kp, sink, gate, dim ** -0.5, heads)
        close(ops.latent_decode(q, uk, uv, cache, lengths, kp, sink, gate, dim ** -0.5, heads), want, dtype)


def test_latent_prep_norms_and_appends():
    from oslo_b200.ops import cuda_ops
    for dtype in DTYPES:
        p = rnd(3, 400, dtype=dtype)
        wq, wk = rnd(128, dtype=dtype), rnd(72, dtype=dtype)
        cache = torch.zeros(3, 9, 72, dtype=dtype, device="cuda")
        lengths = torch.full((3,), 4, dtype=torch.int32, device="cuda")
        got = cuda_ops.latent_prep(p[:, 8:136], wq, p[:, 200:272], wk, cache, lengths, 1e-5)
        close(got, ref.rms_norm(p[:, 8:136], wq, 1e-5), dtype)
        close(cache[:, 4], ref.rms_norm(p[:, 200:272], wk, 1e-5), dtype)
        cache[:, 4] = 0
        assert not cache.any()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,width,ff,experts,top", [(1, 64, 32, 4, 2), (5, 40, 24, 3, 3), (16, 256, 96, 8, 2), (17, 256, 96, 8, 2),
                                                       (200, 128, 300, 5, 1), (300, 36, 20, 7, 3), (700, 512, 256, 16, 4)])
def test_moe(dtype, rows, width, ff, experts, top):
    h = rnd(rows, width, dtype=dtype)
    w, b = rnd(experts, width, dtype=dtype, scale=width ** -0.5), rnd(experts, dtype=dtype)
    up, down = rnd(experts, ff, width, dtype=dtype, scale=width ** -0.5), rnd(experts, width, ff, dtype=dtype, scale=ff ** -0.5, seed=2)
    idx, wgt = ops.moe_route(h, w, b, top)
    ridx, rw = ref.moe_route(h, w, b, top)
    z = h.float() @ w.float().t() + b.float()
    gap = z.topk(min(top + 1, experts), -1).values
    clear = (gap[:, top - 1] - gap[:, -1] > 1e-4) if experts > top else torch.ones(rows, dtype=torch.bool, device="cuda")
    assert torch.equal(idx[clear].sort(-1).values, ridx[clear].sort(-1).values)
    close(wgt.sum(-1), torch.ones(rows, device="cuda"), torch.float32)
    for n in (rows, max(1, min(rows, 8 // top))):                       # the few-rows path and the grouped product
        y, slots = ops.moe_experts(h[:n], idx[:n].contiguous(), up, down)
        y = y[slots.reshape(-1).long()] if slots is not None else y
        close(y, ref.moe_experts(h[:n], idx[:n], up, down), dtype)
    assert rw.shape == wgt.shape


def test_moe_when_one_expert_takes_everything():
    for dtype in (torch.float32, torch.bfloat16):
        h = rnd(600, 64, dtype=dtype)
        up, down = rnd(6, 32, 64, dtype=dtype, scale=0.1), rnd(6, 64, 32, dtype=dtype, scale=0.1, seed=1)
        idx = torch.full((600, 1), 4, dtype=torch.int32, device="cuda")
        y, slots = ops.moe_experts(h, idx, up, down)
        close(y[slots.reshape(-1).long()], ref.moe_experts(h, idx, up, down), dtype)
