"""The kernels behind Dekutar against the fp32 PyTorch statements of the same ops, over sizes that do and do not fit the
vector widths and tiles, and the whole model on the GPU against the plain implementation in ``plain_dekutar.py``."""

import pytest
import torch

import oslo_b200 as ob
from oslo_b200 import ops
from oslo_b200.generation import BatchSteps, GraphedGreedyDecoder
from oslo_b200.models.common import StaticKVCache
from oslo_b200.ops import reference as ref
from oslo_b200.ops.reference import SublayerResult

from . import plain_dekutar as plain
from .dekutar_cases import CASES, attn, case, latent, make_tensors, mlstm, moe, steady, write_model

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


def padding(batch, s, real=1):
    """``keep`` ``[batch, s]`` with padding on the left of every row but the last (at least ``real`` real tokens) and its ``lead``."""
    keep = torch.ones(batch, s, dtype=torch.uint8, device="cuda")
    lead = torch.zeros(batch, dtype=torch.int32, device="cuda")
    for b in range(batch - 1):
        lead[b] = min(s - real, 3 + 14 * b)
        keep[b, :int(lead[b])] = 0
    return keep, lead


# ---------------------------------------------------------------------------------------------------- streams
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,n,cols", [(1, 2, 256), (7, 1, 100), (33, 4, 1024), (5, 3, 37), (70, 2, 512), (3, 8, 4096), (4, 11, 40), (6, 16, 64)])
def test_hyper_join(dtype, rows, n, cols):
    x = rnd(rows, n, cols)
    w_out, mix, w_in, w = rnd(n, dtype=dtype), rnd(n, n, dtype=dtype), rnd(n, dtype=dtype, seed=1), rnd(cols, dtype=dtype, scale=0.3)
    y = rnd(rows, cols + 8, dtype=dtype)[:, :cols]
    top, experts = 3, 4
    g = torch.Generator().manual_seed(rows)
    choice = torch.stack([torch.randperm(experts + 2, generator=g)[:top] for _ in range(rows)]).to(torch.int32).cuda()
    weights = torch.rand(rows, top, generator=g).cuda()
    slots = torch.randperm(rows * top + 5, generator=g)[:rows * top].to(torch.int32).view(rows, top).cuda()
    own, shared, gate = rnd(rows, cols, dtype=dtype, seed=3), rnd(rows, cols + 8, dtype=dtype, seed=4)[:, 8:], rnd(rows, 9, dtype=dtype)[:, 4:5]
    ordered, placed = rnd(rows * top, cols, dtype=dtype), rnd(rows * top + 5, cols, dtype=dtype)
    ordered[(choice >= experts).view(-1)] = float("nan")  # rows of choices that are no expert hold anything
    clean = lambda r: r._replace(y=torch.nan_to_num(r.y))                                       # noqa: E731
    for r in (None, SublayerResult(y), SublayerResult(ordered, None, weights, choice, experts, own),
              SublayerResult(placed, torch.where(choice >= experts, -1, slots), weights, choice, experts, own, shared, gate),
              SublayerResult(placed, slots, weights), SublayerResult(y, shared=shared, shared_gate=gate)):
        for wi, scale in ((w_in, 1.0), (None, 0.4)):
            x1, h1 = ops.hyper_join(x, r, w_out, mix, wi, w, 1e-4, scale)
            x2, h2 = ref.hyper_join(x, None if r is None else clean(r), w_out, mix, wi, w, 1e-4, scale)
            close(x1, x2, torch.float32)                  # the streams are 32-bit whatever the storage type
            close(h1, h2, dtype)
    same = x[:, :1].expand(-1, n, -1)                     # streams that are all equal, held once
    for a, b in zip(ops.hyper_join(same, SublayerResult(y), w_out, mix, w_in, w, 1e-4), ref.hyper_join(same, SublayerResult(y), w_out, mix, w_in, w, 1e-4)):
        close(a, b, dtype if a.dim() == 2 else torch.float32)


# ---------------------------------------------------------------------------------------------------- attention
WINDOWS = [(0, 0), (1, 0), (1, 5), (20, 0), (33, 9), (130, 70), (64, 300), (5000, 3)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("batch,sq,sk,heads,groups,dim,vdim", [
    (2, 50, 50, 4, 1, 64, 64), (1, 2, 9, 4, 2, 24, 16), (2, 33, 70, 6, 3, 48, 80), (1, 140, 500, 4, 2, 128, 128), (2, 300, 300, 2, 1, 64, 64),
    (2, 130, 130, 4, 2, 192, 128), (3, 37, 37, 5, 1, 9, 9), (2, 257, 400, 8, 2, 64, 32), (2, 600, 600, 2, 2, 32, 136)])
def test_windows_and_gates(dtype, batch, sq, sk, heads, groups, dim, vdim):
    q, k, v = (rnd(batch, n, h, d, dtype=dtype, seed=i) for i, (n, h, d) in enumerate(((sq, heads, dim), (sk, groups, dim), (sk, groups, vdim))))
    k[:, 1] *= 4.0                                        # a kept key that stands out
    narrow, wide = rnd(batch * sq, heads + 8, dtype=dtype)[:, :heads], rnd(batch * sq, heads * vdim, dtype=dtype, seed=5)
    keep, lead = padding(batch, sk, sq if sk > sq else 1)
    sink = rnd(heads, dtype=dtype)
    for window, kept in WINDOWS:
        for kp, ld in ((None, None), (keep, lead)):
            for gate, snk in ((None, None), (narrow, None), (wide, sink)):
                args = (q, k, v, kp, snk, gate, dim ** -0.5, 0.0, window, kept, ld)
                want, _ = ref.sink_attention(*args)
                close(ops.sink_attention(*args), want, dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16, torch.float16])
@pytest.mark.parametrize("batch,sq,sk,heads,dim,rot,vdim", [
    (2, 50, 50, 3, 64, 32, 88), (1, 140, 300, 2, 128, 64, 128), (2, 33, 33, 2, 16, 8, 24), (1, 257, 257, 2, 96, 64, 64), (2, 64, 130, 1, 128, 64, 200),
    (1, 40, 40, 2, 192, 64, 128), (1, 30, 30, 2, 256, 64, 64), (2, 29, 29, 3, 7, 6, 5), (1, 200, 200, 4, 64, 64, 64), (1, 1, 9, 2, 64, 32, 64)])
def test_attention_with_a_shared_key_part(dtype, batch, sq, sk, heads, dim, rot, vdim):
    q, k, v = (rnd(batch, n, heads, d, dtype=dtype, seed=i) for i, (n, d) in enumerate(((sq, dim + rot), (sk, dim), (sk, vdim))))
    cache = rnd(batch, sk + 5, 40 + rot, dtype=dtype, seed=4)
    k_rot, gate = cache[:, :sk, 40:], rnd(batch * sq, heads * vdim, dtype=dtype)
    k[:, 0] *= 3.0
    keep, _ = padding(batch, sk, sq if sk > sq else 1)
    for kp in (None, keep):
        args = (q[..., :dim], k, v, kp, None, gate, (dim + rot) ** -0.5, 0.0, 0, 0, None, q[..., dim:], k_rot)
        want, _ = ref.sink_attention(*args)
        close(ops.sink_attention(*args), want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("batch,heads,groups,dim,vdim,tmax,length", [
    (2, 6, 2, 64, 72, 200, 131), (1, 3, 1, 20, 12, 64, 1), (3, 17, 1, 48, 80, 96, 96), (1, 16, 4, 128, 128, 1500, 1400), (9, 2, 1, 9, 11, 33, 20),
    (1, 40, 4, 64, 64, 700, 641), (2, 5, 5, 256, 256, 400, 390), (1, 8, 1, 320, 40, 300, 255), (2, 8, 8, 16, 16, 1100, 1099)])
def test_grouped_decode_in_windows(dtype, batch, heads, groups, dim, vdim, tmax, length):
    from oslo_b200.ops import cuda_ops
    q = rnd(batch, heads, dim, dtype=dtype)
    k, v = rnd(batch, groups, tmax, dim, dtype=dtype), rnd(batch, groups, tmax, vdim, dtype=dtype, seed=2)
    k[:, :, 0] *= 5.0
    k[:, :, length:], v[:, :, length:] = float("nan"), float("nan")        # nothing beyond the valid length may be touched
    lengths = torch.full((batch,), length, dtype=torch.int32, device="cuda")
    keep, lead = padding(batch, length)
    gate, sink = rnd(batch, heads + 4, dtype=dtype)[:, :heads], rnd(heads, dtype=dtype)
    for window, kept in WINDOWS + [(length, 2), (length - 1, 0), (max(1, length - 4), 4)]:
        for kp, ld in ((None, None), (keep, lead)):
            for g, s in ((gate, None), (None, sink)):
                args = (lengths, kp, s, dim ** -0.5, 0.0, g, window, kept, ld)
                want = ref.grouped_decode(q, torch.nan_to_num(k), torch.nan_to_num(v), *args)
                close(cuda_ops.grouped_decode(q, k, v, *args), want, dtype)


def test_windowed_decode_reads_nothing_outside_its_window():
    """Keys and values outside may hold anything, numbers that are none included."""
    from oslo_b200.ops import cuda_ops
    for dtype in DTYPES:
        q, k, v = rnd(2, 4, 64, dtype=dtype), rnd(2, 1, 300, 64, dtype=dtype), rnd(2, 1, 300, 64, dtype=dtype, seed=1)
        lengths = torch.tensor([290, 211], dtype=torch.int32, device="cuda")
        args = (lengths, None, None, 0.125, 0.0, None, 40, 10, None)
        want = ref.grouped_decode(q, k, v, *args)
        for b in range(2):
            for t in (k, v):
                t[b, :, 10:int(lengths[b]) - 40] = float("nan")
                t[b, :, int(lengths[b]):] = float("nan")
        close(cuda_ops.grouped_decode(q, k, v, *args), want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("batch,s,heads,groups,dim,rot", [(2, 9, 6, 2, 64, 32), (1, 1, 4, 1, 128, 128), (3, 5, 5, 5, 9, 6), (2, 3, 3, 1, 40, 0), (1, 7, 2, 1, 320, 320)])
def test_qkv_prep_without_weights_and_with_keys_as_values(dtype, batch, s, heads, groups, dim, rot):
    from oslo_b200.ops import cuda_ops
    n, past, tmax = batch * s, 4, s + 9
    p = rnd(n, (heads + groups) * dim + 8, dtype=dtype)
    q, k = p[:, :heads * dim], p[:, heads * dim:(heads + groups) * dim]
    pos = torch.stack([torch.arange(past, past + s) + 1000 * b for b in range(batch)]).cuda()
    freq = torch.tensor(ref.rotary_frequencies(rot, 5e4), device="cuda")
    kc, vc = (torch.zeros(batch, groups, tmax, dim, dtype=dtype, device="cuda") for _ in range(2))
    lengths = torch.full((batch,), past, dtype=torch.int32, device="cuda")
    got = cuda_ops.qkv_prep(q, k, k, None, None, 1e-4, pos, freq, kc, vc, lengths)
    close(got, ref.norm_rotate(q.reshape(batch, s, heads, dim), None, 1e-4, pos, freq), dtype)
    close(kc[:, :, past:past + s].transpose(1, 2), ref.norm_rotate(k.reshape(batch, s, groups, dim), None, 1e-4, pos, freq), dtype)
    assert torch.equal(vc[:, :, past:past + s].transpose(1, 2), k.reshape(batch, s, groups, dim))


# ---------------------------------------------------------------------------------------------------- latents
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("batch,s,q_rank,rank,rot,heads,dim", [(2, 9, 96, 64, 32, 3, 24), (1, 1, 24, 512, 64, 2, 128), (3, 5, 13, 9, 6, 5, 7), (4, 40, 128, 72, 8, 1, 16)])
def test_latent_prep_and_rotation_in_place(dtype, batch, s, q_rank, rank, rot, heads, dim):
    from oslo_b200.ops import cuda_ops
    n, past, tmax = batch * s, 3, s + 8
    p = rnd(n, q_rank + rank + rot + 16, dtype=dtype)
    cq, ckv = p[:, 8:8 + q_rank], p[:, 8 + q_rank:8 + q_rank + rank + rot]
    wq, wk = rnd(q_rank, dtype=dtype), rnd(rank, dtype=dtype, seed=1)
    pos = torch.stack([torch.arange(past, past + s) + 900 * b for b in range(batch)]).cuda()
    freq = torch.tensor(ref.rotary_frequencies(rot, 3e5), device="cuda")
    lengths = torch.full((batch,), past, dtype=torch.int32, device="cuda")
    cache = torch.zeros(batch, tmax, rank + rot, dtype=dtype, device="cuda")
    for rows in (False, True):
        cache.zero_()
        got, c = cuda_ops.latent_prep(cq, wq, ckv, wk, cache, lengths, 1e-4, pos, freq, rows)
        close(got, ref.rms_norm(cq, wq, 1e-4), dtype)
        want = ref.rms_norm(ckv[:, :rank], wk, 1e-4).view(batch, s, rank)
        close(cache[:, past:past + s, :rank], want, dtype)
        close(cache[:, past:past + s, rank:], ref.rotate_halves(ckv[:, rank:].reshape(batch, s, 1, rot), pos, freq)[:, :, 0], dtype)
        assert c.size(0) == (n if rows else 0) and (not rows or torch.equal(c.view(batch, s, rank), cache[:, past:past + s, :rank]))
        cache[:, past:past + s] = 0
        assert not cache.any()
    q = rnd(batch, s, heads, dim + rot, dtype=dtype)
    want = torch.cat([q[..., :dim], ref.rotate_halves(q[..., dim:], pos, freq)], dim=-1)
    assert cuda_ops.rotate_halves_(q, pos, freq).data_ptr() == q.data_ptr()
    close(q, want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("batch,heads,dim,rot,vdim,rank,tmax,length", [
    (1, 5, 64, 32, 72, 96, 200, 131), (5, 20, 128, 64, 128, 512, 300, 290), (3, 2, 16, 16, 24, 32, 64, 1), (2, 3, 7, 6, 5, 9, 70, 60),
    (4, 33, 32, 16, 40, 96, 150, 149), (17, 2, 48, 8, 16, 64, 90, 80), (1, 2, 8, 2, 8, 700, 50, 49)])
def test_latent_decode(dtype, batch, heads, dim, rot, vdim, rank, tmax, length):
    q = rnd(batch, heads * (dim + rot), dtype=dtype)
    uk, uv = rnd(heads * dim, rank, dtype=dtype, scale=rank ** -0.5), rnd(heads * vdim, rank, dtype=dtype, scale=rank ** -0.5)
    cache = rnd(batch, tmax, rank + rot, dtype=dtype)
    cache[:, 0] *= 3.0
    lengths = torch.full((batch,), length, dtype=torch.int32, device="cuda")
    lengths[0] = max(1, length - 3)
    pos = (lengths - 1).long()[:, None]
    freq = torch.tensor(ref.rotary_frequencies(rot, 100.0), device="cuda")
    keep, _ = padding(batch, length, 4 if length > 4 else 1)
    sink = rnd(heads, dtype=dtype)
    for kp in (None, keep):
        for gate, snk in ((rnd(batch, heads * vdim, dtype=dtype), None), (rnd(batch, heads, dtype=dtype), sink)):
            args = (lengths, kp, snk, gate, (dim + rot) ** -0.5, heads, pos, freq)
            want = ref.latent_decode(q, uk, uv, cache, *args)
            got = ops.latent_decode(q, uk, uv, cache, *args)
            close(got, want, dtype)


# ---------------------------------------------------------------------------------------------------- matrix memory
def memory_inputs(batch, s, heads, dim, vdim, dtype, width=40):
    n = batch * s
    p = rnd(n, 2 * heads * dim + heads * vdim + 8, dtype=dtype)
    q, k, v = p[:, :heads * dim], p[:, heads * dim:2 * heads * dim], p[:, 2 * heads * dim:2 * heads * dim + heads * vdim]
    return q, k, v, rnd(n, 2 * heads, scale=6.0), rnd(2 * heads, dtype=dtype, scale=3.0)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("batch,s,heads,dim,vdim", [(2, 37, 3, 40, 72), (1, 1, 2, 16, 8), (1, 200, 1, 12, 20), (2, 17, 2, 100, 33), (1, 150, 2, 128, 128),
                                                    (3, 50, 1, 256, 24), (1, 9, 1, 300, 40), (2, 64, 2, 64, 64), (1, 40, 1, 16, 511)])
def test_matrix_memory(dtype, batch, s, heads, dim, vdim):
    q, k, v, z, bias = memory_inputs(batch, s, heads, dim, vdim, dtype)
    ext = ops.load_ext(required=True)
    wide = ref.memory_state_width(vdim)
    s0, m0 = rnd(batch, heads, dim, wide, scale=0.5), rnd(batch, heads)
    s0[..., vdim + 1:] = 0
    keep, _ = padding(batch, s)
    for cap in (2.0, 15.0):
        for kp in (None, keep):
            for start in (None, (s0, m0)):
                o, nq, m, end, top = ref.matrix_memory(q, k, v, z, bias, cap, kp, *(start or (None, None)), batch, heads)
                for chunks in (0, 1, 2, 5):
                    st, tp = (t.clone() if start else torch.zeros_like(t) for t in (s0, m0))
                    read, write, begin, m2 = ext.memory_gates(z, bias, cap, kp, tp, batch)
                    o2, nq2 = ext.memory_recurrence(q, k, v, read, write, begin, dim ** -0.5, kp, st, batch, heads, dim, vdim, chunks)
                    close(m2, m, torch.float32)
                    close(o2, o, torch.float32, 2.0)
                    close(nq2, nq, torch.float32, 2.0)
                    close(st[..., :vdim + 1], end[..., :vdim + 1], torch.float32, 2.0)
                    close(tp, top, torch.float32)


def test_matrix_memory_with_gates_of_every_size():
    """Forget gates from 0 to 1, input gates that swamp or vanish: the periods in which the state is kept relative differ, the result
    does not. More tokens than one pass of the gate scan covers."""
    for f, i, s in ((-60.0, 0.0, 90), (-9.0, 0.0, 90), (-3.0, 5.0, 90), (0.0, -20.0, 90), (3.0, 3.0, 90), (30.0, 0.0, 90), (4.0, 0.0, 4500)):
        q, k, v, z, _ = memory_inputs(1, s, 2, 16, 12, torch.float32)
        z = 0.5 * z
        bias = torch.tensor([i, i, f, f], device="cuda")
        o, nq, m, end, top = ref.matrix_memory(q, k, v, z, bias, 80.0, None, None, None, 1, 2)
        for n in ([s], [s // 3, s - s // 3 - 7, 7]):
            st, tp, at, outs = torch.zeros_like(end), torch.zeros_like(top), 0, []
            for c in n:
                outs.append(ops.matrix_memory(*(t[at:at + c] for t in (q, k, v, z)), bias, 80.0, None, st, tp, 1, 2))
                at += c
            for got, want in zip((torch.cat(t) for t in zip(*outs)), (o, nq, m)):
                close(got, want, torch.float32, 4.0)
            close(st, end, torch.float32, 4.0)
            close(tp, top, torch.float32)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("batch,heads,dim,vdim,width", [(1, 5, 40, 72, 200), (5, 3, 20, 30, 37), (2, 16, 128, 128, 1024), (70, 2, 64, 256, 64),
                                                        (1, 1, 7, 2100, 8), (3, 2, 16, 5, 1)])
def test_memory_step_is_one_token_of_the_recurrence(dtype, batch, heads, dim, vdim, width):
    from oslo_b200.ops import cuda_ops
    q, k, v, _, bias = memory_inputs(batch, 1, heads, dim, vdim, dtype)
    x, w = rnd(batch, width + 8, dtype=dtype)[:, :width], rnd(2 * heads, width, dtype=dtype, scale=width ** -0.5)
    nw, gate = rnd(heads * vdim, dtype=dtype), rnd(batch, heads * vdim, dtype=dtype, seed=4)
    s0, m0 = rnd(batch, heads, dim, ref.memory_state_width(vdim)), rnd(batch, heads)
    s0[..., vdim + 1:] = 0
    z = x.float() @ w.float().t()
    for keep in (None, (torch.arange(batch, device="cuda") % 2 == 0).to(torch.uint8)[:, None]):
        o, nq, m, end, top = ref.matrix_memory(q, k, v, z, bias, 9.0, keep, s0, m0, batch, heads)
        st, tp = s0.clone(), m0.clone()
        got = cuda_ops.memory_step(q, k, v, x, w, bias, 9.0, gate, nw, keep, st, tp, 1e-4, heads)
        close(got, ref.gated_rms_norm(o, nw, gate, 1e-4, vdim, "sigmoid", (nq, m)), dtype)
        close(st, end, torch.float32, 2.0)
        close(tp, top, torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,groups,group", [(1, 3, 64), (70, 2, 128), (5, 7, 9), (3, 1, 2048), (11, 2, 700)])
def test_gated_rms_norm_with_a_normaliser(dtype, rows, groups, group):
    n = groups * group
    o, w, gate = rnd(rows, n), rnd(n, dtype=dtype), rnd(rows, n + 8, dtype=dtype)[:, :n]
    both = rnd(rows, groups, seed=1), rnd(rows, groups, scale=3.0, seed=2)
    close(ops.gated_rms_norm(o, w, gate, 1e-3, group, "sigmoid", both), ref.gated_rms_norm(o, w, gate, 1e-3, group, "sigmoid", both), dtype)


# ---------------------------------------------------------------------------------------------------- experts
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width,outputs,top", [(1, 256, 20, 4), (7, 100, 6, 6), (64, 37, 5, 1), (65, 64, 33, 8), (300, 128, 300, 5), (200, 30, 12, 3), (90, 64, 35, 4)])
def test_scored_routing(dtype, rows, width, outputs, top):
    h, w = rnd(rows, width + 8, dtype=dtype)[:, :width], rnd(outputs, width, dtype=dtype, scale=2.0 * width ** -0.5)
    corr = rnd(outputs, dtype=dtype, scale=0.05)
    if width % 8:
        h = h.contiguous()
    idx, weights = ops.moe_route(h, w, corr, top, scored=True)
    want_idx, want = ref.moe_route(h, w, corr, top, scored=True)
    score = torch.softmax(h.float() @ w.float().t(), -1) + corr.float()
    # equal choices up to close calls
    assert torch.allclose(score.gather(1, idx.long()), score.gather(1, want_idx.long()), atol=1e-5)
    same = (idx == want_idx).all(1)
    assert same.float().mean() > 0.9
    close(weights[same], want[same], torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width,ff,experts,identity,top", [(1, 64, 24, 4, 2, 3), (2, 48, 96, 6, 3, 4), (40, 64, 40, 5, 2, 4), (300, 128, 64, 8, 4, 3),
                                                                (33, 35, 13, 3, 2, 2), (2, 35, 7, 3, 5, 4), (70, 256, 256, 1, 1, 2), (50, 40, 136, 3, 0, 3)])
def test_gated_experts_and_choices_that_are_none(dtype, rows, width, ff, experts, identity, top):
    g = torch.Generator().manual_seed(rows)
    h, up, down = rnd(rows, width, dtype=dtype), rnd(experts, 2 * ff, width, dtype=dtype, scale=width ** -0.5), rnd(experts, width, ff, dtype=dtype, scale=ff ** -0.5)
    for only_identity in (False, True):
        if only_identity and identity < top:
            continue
        pick = lambda: experts + torch.randperm(identity, generator=g)[:top] if only_identity else torch.randperm(experts + identity, generator=g)[:top]  # noqa: E731
        idx = torch.stack([pick() for _ in range(rows)]).to(torch.int32).cuda()
        y, slots = ops.moe_experts(h, idx, up, down, "silu")
        want = ref.moe_experts(h, idx, up, down, "silu").view(rows, top, width)
        own = idx < experts
        at = torch.arange(rows * top, device="cuda").view(rows, top) if slots is None else slots.long()
        assert slots is None or bool((slots[~own] == -1).all())
        if bool(own.any()):
            close(y[at[own]], want[own], dtype)


# ---------------------------------------------------------------------------------------------------- the whole model
MODEL_TOL = 1e-4   # 32-bit
WIDE = {
    # chunked recurrences, several key tiles, cluster sizes above 1, more than one tile of query heads per key head, routed batches
    "wide": case(200, 272, 1e-6, 3, mlstm(4, 128, 64, 10.0, moe(88, 18, 3, 5, 136)), attn(20, 1, 64, 0.12, 140, 10, 32, moe(64, 8, 2, 2, 64)),
                 latent(4, 128, 64, 128, 96, 128, 0.07, moe(128, 8, 4, 4, 96), 1e4), mlstm(2, 64, 256, 6.0, None),
                 attn(4, 2, 128, 0.1, 30, 150, 128, None, 5e5), latent(20, 64, 32, 64, 128, 96, 0.1, None)),
}
ALL = {**{k: v for k, v in CASES.items() if k != "ones"}, **WIDE}


def load(tmp_path, cfg, tensors=None, dtype=torch.float32):
    if tensors is None:
        tensors = make_tensors(cfg) if dtype == torch.float32 else steady(make_tensors(cfg))
    write_model(str(tmp_path), cfg, tensors)
    model = ob.load_causal_lm(str(tmp_path), torch_dtype=dtype).cuda().fuse().eval()
    return model, tensors


def ids(n, vocab, seed=1):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def apart(a, b):
    """Per position: root mean square over the vocabulary, relative to the logits' own."""
    return (a - b).pow(2).mean(-1).sqrt() / b.pow(2).mean().sqrt()


class Want:
    """The plain model's logits of a sequence and, per position, how far weights off by a fraction of a 16-bit step move them."""

    def __init__(self, cfg, tensors, seq, dtype):
        self.logits = plain.forward(cfg, tensors, seq)
        self.noise = torch.zeros(len(seq), dtype=torch.float64)
        g = torch.Generator().manual_seed(77)
        for _ in range(0 if dtype == torch.float32 else 2):
            off = {k: t.double() * (1 + 2.0 ** -9 * torch.randn(t.shape, generator=g)) for k, t in tensors.items()}
            self.noise = torch.maximum(self.noise, apart(plain.forward(cfg, off, seq), self.logits))


def same(got, want, dtype, at=slice(None), factor=1.0):
    """In 32-bit every position counts; in 16-bit the tolerance follows what rounding does there, and one position in thirty may be one
    that it blows up all the same (a router's close call)."""
    got = got.double().cpu()
    assert torch.isfinite(got).all() and got.shape == want.logits[at].shape
    d = (got - want.logits[at]).pow(2).mean(-1).sqrt() / want.logits.pow(2).mean().sqrt()
    if dtype == torch.float32:
        assert float(d.max()) < factor * MODEL_TOL, float(d.max())
        return
    noise = want.noise[at]
    over = int((d > factor * (0.02 + 4.0 * noise)).sum())
    assert over <= -(-d.numel() // 30) and float(d.median()) < factor * (0.01 + 2.0 * float(noise.median())), (over, d, noise)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", sorted(ALL))
def test_model_prompts_decoding_and_portions(tmp_path, dtype, name):
    cfg = ALL[name]
    model, tensors = load(tmp_path, cfg, dtype=dtype)
    n = 200 if name == "wide" else 70
    seq = ids(n, cfg["vocab"])
    want = Want(cfg, tensors, seq, dtype)
    x = torch.tensor([seq], device="cuda")
    before = ops.load_ext(required=True).launch_count()
    with torch.no_grad():
        same(model(input_ids=x).logits[0], want, dtype)
        same(model(input_ids=x, use_cache=False).logits[0], want, dtype)
        assert ops.load_ext().launch_count() > before
        for portions in ([n - 12] + [1] * 12, [1] * 20, [2] * 6 + [n - 13, 1], [n // 2, 2, n - n // 2 - 2]):
            cache, at, got = StaticKVCache(16, grow=True), 0, []
            for m in portions:
                got.append(model(input_ids=x[:, at:at + m], past_key_values=cache, use_cache=True).logits[0])
                at += m
            same(torch.cat(got), want, dtype, slice(0, at))
    assert int(ops.load_ext().error_word(x).item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_model_batches_of_unequal_requests(tmp_path, dtype, name):
    cfg = ALL[name]
    model, tensors = load(tmp_path, cfg, dtype=dtype)
    lens, tails = (40, 1, 23, 150), (6, 9, 3, 2)
    seqs = [ids(a + b, cfg["vocab"], seed=a) for a, b in zip(lens, tails)]
    want = [Want(cfg, tensors, s, dtype) for s in seqs]
    steps = BatchSteps(model, reserve=1)
    out = steps.start([s[:a] for s, a in zip(seqs, lens)])
    got = [[out[r, steps.pad[r]:]] for r in range(4)]
    live, at = [0, 1, 2, 3], list(lens)
    while True:
        rows = [i for i, r in enumerate(live) if at[r] < len(seqs[r])]
        if not rows:
            break
        steps.keep(rows)
        live = [live[i] for i in rows]
        out = steps.advance([seqs[r][at[r]] for r in live])
        for i, r in enumerate(live):
            got[r].append(out[i])
            at[r] += 1
    for r in range(4):
        same(torch.cat(got[r]), want[r], dtype)


def test_model_many_rows_decode_like_few(tmp_path):
    cfg = WIDE["wide"]
    model, tensors = load(tmp_path, cfg, dtype=torch.bfloat16)
    seqs = [ids(34, 200, seed=s) for s in range(21)]
    want = [Want(cfg, tensors, s, torch.bfloat16) for s in seqs[:3]]
    x = torch.tensor(seqs, device="cuda")
    cache = StaticKVCache(40)
    with torch.no_grad():
        model(input_ids=x[:, :26], past_key_values=cache)
        got = torch.cat([model(input_ids=x[:, t:t + 1], past_key_values=cache).logits for t in range(26, 34)], dim=1)
    for r in range(3):
        same(got[r], want[r], torch.bfloat16, slice(26, 34))


def fed(model, seq, prompt):
    x, cache = torch.tensor([seq], device="cuda"), StaticKVCache(len(seq))
    with torch.no_grad():
        out = [model(input_ids=x[:, :prompt], past_key_values=cache).logits[0]]
        out += [model(input_ids=x[:, t:t + 1], past_key_values=cache).logits[0] for t in range(prompt, len(seq))]
    return torch.cat(out)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim", [16, 64])
def test_model_keys_at_the_edges_of_a_window(tmp_path, dtype, dim):
    """A changed token moves the positions that see it and leaves the others as they are, to the bit."""
    size, kept, n = 150, 130, 420
    cfg = case(64, 64, 1e-6, 2, attn(2, 1, dim, 0.5 / dim, size, kept, 4, None, 1e5))
    model, tensors = load(tmp_path, cfg, dtype=dtype)
    seq = [t % 60 for t in ids(n, 60, 8)]
    want = Want(cfg, tensors, seq, dtype)
    for prompt in (n, 300):
        got = fed(model, seq, prompt)
        same(got, want, dtype)
        for at in (0, 127, 128, kept - 1, kept, 149, 150, 255, 256, 299, 300):
            other = list(seq)
            other[at] = 61
            moved = (fed(model, other, prompt) - got).abs().amax(-1)
            assert not any(bool(moved[i]) for i in range(n) if not plain.sees(i, at, size, kept)), (prompt, at)
            sees = [i for i in range(n) if plain.sees(i, at, size, kept)]
            assert float((moved[sees] > 0).float().mean()) > 0.95, (prompt, at)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_model_far_keys_of_latent_attention(tmp_path, dtype):
    cfg = case(64, 64, 1e-6, 2, latent(4, 64, 32, 64, 64, 64, 0.15, None, 1e6), mlstm(1, 16, 16, 4.0, None))
    tensors = make_tensors(cfg, 3)
    for name in ("l0.mix.uq", "l0.mix.uk"):
        tensors[name] = tensors[name] * 1.5
    seq = [t % 60 for t in ids(420, 60, 8)]
    for at in (0, 1, 127, 128, 255):
        seq[at] = 63
    want = Want(cfg, tensors, seq, dtype)
    other = plain.forward(cfg, tensors, [62] + seq[1:])
    model, _ = load(tmp_path, cfg, tensors, dtype)
    same(model(input_ids=torch.tensor([seq], device="cuda")).logits[0].detach(), want, dtype, factor=2.0)
    same(fed(model, seq, 400), want, dtype, factor=2.0)
    moved = (other[400:] - want.logits[400:]).pow(2).mean(-1).sqrt().max() / want.logits.pow(2).mean().sqrt()
    assert float(moved) > 20 * MODEL_TOL   # the first token is seen from the end


@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_model_greedy_generation_and_captured_decoding(tmp_path, name):
    cfg = ALL[name]
    model, tensors = load(tmp_path, cfg)
    prompts = [ids(9, cfg["vocab"], 11), ids(9, cfg["vocab"], 12)]
    want = []
    for p in prompts:
        seq = list(p)
        for _ in range(10):
            seq.append(int(plain.forward(cfg, tensors, seq)[-1].argmax()))
        want.append(seq)
    want = torch.tensor(want)
    x = torch.tensor(prompts, device="cuda")
    kw = dict(max_new_tokens=10, eos_token_id=None, pad_token_id=None)
    assert torch.equal(model.generate(x, **kw).cpu(), want)
    assert torch.equal(model.generate(x, cuda_graph=True, **kw).cpu(), want)
    dec = GraphedGreedyDecoder(model, max_len=32)
    for _ in range(2):                                    # the captured step, the cache and the states are used again
        assert torch.equal(dec.generate(x, 10).cpu(), want)
    assert dec.replays > 0
    # the 16-bit model decodes the same tokens eagerly and from the captured step
    half, _ = load(tmp_path, cfg, dtype=torch.bfloat16)
    assert torch.equal(half.generate(x, **kw), half.generate(x, cuda_graph=True, **kw))


def test_model_with_sizes_beyond_one_kernel(tmp_path):
    cfg = case(40, 32, 1e-5, 9, mlstm(1, 600, 24, 8.0, moe(8, 3, 70, 66, 16)), attn(2, 1, 300, 0.06, 9, 4, 300, None), latent(2, 200, 100, 24, 16, 1100, 0.05, None))
    model, tensors = load(tmp_path, cfg)
    seq = ids(24, 40)
    want = Want(cfg, tensors, seq, torch.float32)
    x = torch.tensor([seq], device="cuda")
    cache = StaticKVCache(24)
    with torch.no_grad():
        got = [model(input_ids=x[:, a:b], past_key_values=cache).logits[0] for a, b in ((0, 15), (15, 20), (20, 21), (21, 22))]
    same(torch.cat(got), want, torch.float32, slice(0, 22), 2.0)


def test_long_decoding_keeps_agreeing_with_the_prompt_form(tmp_path):
    cfg = CASES["heads64"]
    for dtype in (torch.float32, torch.bfloat16):
        model, tensors = load(tmp_path, cfg, dtype=dtype)
        seq = ids(300, 128, 5)
        want = Want(cfg, tensors, seq, dtype)
        same(fed(model, seq, 3), want, dtype, factor=1.5)
