"""The kernels behind Begovik against the fp32 PyTorch statements of the same ops, over sizes that do and do not fit the
vector widths and tiles, and the whole model on the GPU against the plain implementation in ``plain_begovik.py``."""

import pytest
import torch

import oslo_b200 as ob
from oslo_b200 import ops
from oslo_b200.generation import BatchSteps, GraphedGreedyDecoder
from oslo_b200.models.common import StaticKVCache
from oslo_b200.ops import reference as ref

from . import plain_begovik as plain
from .begovik_cases import CASES, attn, case, dense, far_key_weights, lin, make_tensors, mamba, parallel, wkv, write_model

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


def some_padding(batch, s):
    """The last row as it is, the others with padding on the left."""
    keep = torch.ones(batch, s, dtype=torch.uint8, device="cuda")
    for b in range(batch - 1):
        keep[b, :min(s - 1, 3 + 14 * b)] = 0
    return keep


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,cols", [(1, 256), (7, 100), (33, 1024), (5, 37), (129, 512), (3, 4096)])
def test_branch_join(dtype, rows, cols):
    x = rnd(rows, cols)
    ys = [rnd(rows, cols + 8, dtype=dtype, seed=i, scale=1.0 + i)[:, :cols] for i in range(3)]
    ws = [rnd(cols, dtype=dtype, seed=9 + i) for i in range(4)]
    for branches in ([(ys[0], None, 1.0)], [(ys[0], None, 1.0), (ys[1], None, 1.0)],
                     [(ys[0], ws[0], 0.5), (ys[1], ws[1], 0.5), (ys[2], None, 1.0)], [(ys[2], ws[1], 0.5), (ys[1], ws[0], 0.5)]):
        for nxt in ([], [ws[2]], [ws[2], ws[3]]):
            x1, h1 = ops.branch_join(x, branches, 0.3, 1e-4, nxt)
            x2, h2 = ref.branch_join(x, branches, 0.3, 1e-4, nxt)
            assert x1.dtype == torch.float32 and len(h1) == len(nxt)
            close(x1, x2, torch.float32)                  # the stream is 32-bit whatever the storage type
            for a, b in zip(h1, h2):
                close(a, b, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cols", [96, 50, 2048])
def test_clamped_glu(dtype, cols):
    t = rnd(9, 2 * cols + 8, dtype=dtype, scale=2.0)
    for limit in (0.5, 7.0):
        close(ops.clamped_glu(t[:, :cols], t[:, cols:2 * cols], limit, 1.702), ref.clamped_glu(t[:, :cols], t[:, cols:2 * cols], limit, 1.702), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,groups,group", [(1, 3, 64), (70, 2, 128), (5, 7, 9), (3, 1, 2048), (11, 2, 700), (9, 4, 24)])
def test_gated_rms_norm(dtype, rows, groups, group):
    n = groups * group
    o, w, gate = rnd(rows, n), rnd(n, dtype=dtype), rnd(rows, n + 8, dtype=dtype)[:, :n]
    for act in ("sigmoid", "silu"):
        close(ops.gated_rms_norm(o, w, gate, 1e-3, group, act), ref.gated_rms_norm(o, w, gate, 1e-3, group, act), dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("batch,s,heads,dim,vdim", [(2, 37, 3, 40, 72), (1, 1, 2, 16, 8), (1, 200, 1, 12, 20), (2, 17, 2, 100, 33),
                                                    (1, 150, 2, 128, 128), (3, 50, 1, 256, 24), (1, 9, 1, 300, 40), (2, 64, 2, 64, 64)])
def test_recurrences_with_decays_of_their_own(dtype, batch, s, heads, dim, vdim):
    n = batch * s
    p = rnd(n, 2 * heads * dim + heads * vdim + 8, dtype=dtype)
    q, k, v = p[:, :heads * dim], p[:, heads * dim:2 * heads * dim], p[:, 2 * heads * dim:2 * heads * dim + heads * vdim]
    ext = ops.load_ext(required=True)
    s0 = rnd(batch, heads, dim, vdim, scale=0.5)
    z, w0, u = rnd(n, heads * dim, scale=2.0), rnd(heads * dim, dtype=dtype) - 2.0, rnd(heads * dim, dtype=dtype)
    decay = torch.tensor([0.999, 0.3, 0.0, 1e-3, 0.05, 1.0][:heads], device="cuda")
    for kp in (None, some_padding(batch, s)):
        for start in (None, s0):
            for name in ("decayed", "bonus"):
                if name == "decayed":
                    want, end = ref.decayed_attention(q, k, v, decay, kp, start, batch, heads)
                    run = lambda st, ch: ext.decayed_recurrence(q, k, v, decay, kp, st, batch, heads, dim, vdim, ch)           # noqa: E731
                else:
                    want, end = ref.bonus_recurrence(q, k, v, z, w0, u, kp, start, batch, heads)
                    run = lambda st, ch: ext.bonus_recurrence(q, k, v, z, w0, u, kp, st, batch, heads, dim, vdim, ch)          # noqa: E731
                for chunks in (0, 1, 2, 5):
                    if name == "bonus" and dim > 256:     # blocks of key channels
                        st = start.clone() if start is not None else torch.zeros_like(s0)
                        got = ops.bonus_recurrence(q, k, v, z, w0, u, kp, st, batch, heads).view(want.shape)
                    else:
                        st = start.clone() if start is not None else torch.zeros_like(s0)
                        got = run(st, chunks)
                    close(got, want, torch.float32, 2.0)
                    close(st, end, torch.float32, 2.0)


def test_every_decay_keeps_its_precision_in_the_scaled_form():
    """Decays from 0 to 1: the periods within which the state is kept relative differ, the result does not."""
    ext = ops.load_ext(required=True)
    for d in (0.0, 1e-30, 1e-9, 1e-4, 0.01, 0.1, 0.12, 0.5, 0.9, 0.9999, 1.0):
        q, k, v = (rnd(1 * 100, 32, seed=i) for i in range(3))
        decay = torch.tensor([d, d], device="cuda")
        st, want = torch.zeros(1, 2, 16, 16, device="cuda"), None
        want, end = ref.decayed_attention(q, k, v, decay, None, None, 1, 2)
        for chunks in (1, 3):
            st.zero_()
            close(ext.decayed_recurrence(q, k, v, decay, None, st, 1, 2, 16, 16, chunks), want, torch.float32)
            close(st, end, torch.float32)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("batch,heads,dim,vdim,rank", [(1, 5, 40, 72, 24), (5, 3, 20, 30, 7), (2, 16, 128, 128, 64), (70, 2, 64, 256, 33),
                                                       (1, 1, 7, 2100, 1)])
def test_steps_are_one_token_of_the_recurrences(dtype, batch, heads, dim, vdim, rank):
    from oslo_b200.ops import cuda_ops
    p = rnd(batch, 2 * heads * dim + heads * vdim + 8, dtype=dtype)
    q, k, v = p[:, :heads * dim], p[:, heads * dim:2 * heads * dim], p[:, 2 * heads * dim:2 * heads * dim + heads * vdim]
    s0 = rnd(batch, heads, dim, vdim)
    decay = torch.linspace(0.0, 1.0, heads, device="cuda")
    t, w2 = rnd(batch, rank, dtype=dtype), rnd(heads * dim, rank, dtype=dtype, scale=rank ** -0.5)
    w0, u = rnd(heads * dim, dtype=dtype) - 1.0, rnd(heads * dim, dtype=dtype)
    nw, gate = rnd(heads * vdim, dtype=dtype), rnd(batch, heads * vdim, dtype=dtype, seed=4)
    z = torch.tanh(t.float()).to(dtype).float() @ w2.float().t()
    for keep in (None, (torch.arange(batch, device="cuda") % 2 == 0).to(torch.uint8)[:, None]):
        want, end = ref.decayed_attention(q, k, v, decay, keep, s0, batch, heads)
        st = s0.clone()
        close(ops.decayed_attention(q, k, v, decay, keep, st, batch, heads), want.view(batch, -1), torch.float32)
        close(st, end, torch.float32)
        want, end = ref.bonus_recurrence(q, k, v, z, w0, u, keep, s0, batch, heads)
        st = s0.clone()
        got = cuda_ops.bonus_step(q, k, v, t, w2, w0, u, nw, gate, keep, st, 1e-5, heads)
        close(got, ref.gated_rms_norm(want.view(batch, -1), nw, gate, 1e-5, vdim, "silu"), dtype)
        close(st, end, torch.float32, 2.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("batch,s,width", [(1, 1, 64), (2, 40, 100), (3, 17, 37), (1, 16, 1024)])
def test_token_shift(dtype, batch, s, width):
    h, mu = rnd(batch * s, width + 8, dtype=dtype)[:, :width], torch.rand(5, width, device="cuda").to(dtype)
    start = rnd(batch, width)
    for kp in (None, some_padding(batch, s)):
        for prev in (None, start):
            want, last = ref.token_shift(h, mu, batch, kp, prev)
            st = prev.clone() if prev is not None else torch.zeros_like(start)
            close(ops.token_shift(h, mu, batch, kp, st), want, dtype)
            close(st, last, torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("batch,s,channels,taps", [(1, 1, 64, 4), (2, 40, 100, 4), (3, 17, 37, 4), (2, 2, 64, 4), (1, 50, 40, 3), (2, 33, 24, 1),
                                                   (1, 70, 32, 21), (1, 3, 9, 7)])
def test_causal_conv(dtype, batch, s, channels, taps):
    x = rnd(batch * s, channels + 8, dtype=dtype)[:, :channels]
    w, b = rnd(channels, taps, dtype=dtype, scale=taps ** -0.5), rnd(channels, dtype=dtype)
    start = rnd(batch, taps - 1, channels)
    for kp in (None, some_padding(batch, s)):
        for prev in (None, start):
            want, last = ref.causal_conv(x, w, b, batch, kp, prev, silu=True)
            st = prev.clone() if prev is not None else torch.zeros_like(start)
            close(ops.causal_conv(x, w, b, batch, kp, st, silu=True), want, dtype)
            if taps > 1:
                close(st, last, torch.float32)


def scan_inputs(n, channels, states, dtype):
    x, z = rnd(n, channels + 8, dtype=dtype)[:, :channels], rnd(n, channels, dtype=dtype, seed=1)
    dt, bias = rnd(n, channels, scale=2.0), rnd(channels, dtype=dtype) - 2.0
    a_log = (torch.rand(channels, states, generator=torch.Generator().manual_seed(3)) * 3.0 - 1.0).to(dtype).cuda()
    bc = rnd(n, 2 * states + 5, dtype=dtype)
    return x, dt, bias, a_log, bc[:, :states], bc[:, states + 2:2 * states + 2], rnd(channels, dtype=dtype, seed=2), z


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("batch,s,channels,states", [(2, 37, 72, 16), (1, 1, 8, 1), (1, 200, 20, 5), (2, 50, 130, 24), (1, 150, 256, 64),
                                                     (3, 20, 33, 100), (1, 19, 16, 256), (2, 64, 512, 8)])
def test_selective_scan(dtype, batch, s, channels, states):
    args = scan_inputs(batch * s, channels, states, dtype)
    ext = ops.load_ext(required=True)
    start = rnd(batch, channels, states, scale=0.5)
    for kp in (None, some_padding(batch, s)):
        for s0 in (None, start):
            want, end = ref.selective_scan(*args, batch, kp, s0)
            real = torch.ones(batch * s, dtype=torch.bool, device="cuda") if kp is None else kp.view(-1).bool()
            for chunks in (0, 1, 2, 5):
                st = s0.clone() if s0 is not None else torch.zeros_like(start)
                got = ext.selective_scan(*args, batch, kp, st, chunks)
                close(got[real], want[real], dtype)
                close(st, end, torch.float32, 2.0)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("batch,channels,states,rank", [(1, 72, 16, 8), (9, 40, 24, 5), (70, 256, 16, 128), (3, 33, 7, 33)])
def test_scan_step_is_one_token_of_the_scan(dtype, batch, channels, states, rank):
    from oslo_b200.ops import cuda_ops
    x, _, bias, a_log, b, c, d, z = scan_inputs(batch, channels, states, dtype)
    low, w = rnd(batch, rank, dtype=dtype), rnd(channels, rank, dtype=dtype, scale=rank ** -0.5)
    dt = low.float() @ w.float().t()
    s0 = rnd(batch, channels, states)
    for keep in (None, (torch.arange(batch, device="cuda") % 2 == 0).to(torch.uint8)[:, None]):
        want, end = ref.selective_scan(x, dt, bias, a_log, b, c, d, z, batch, keep, s0)
        st = s0.clone()
        close(cuda_ops.scan_step(x, low, w, bias, a_log, b, c, d, z, keep, st), want, dtype)
        close(st, end, torch.float32, 2.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("batch,s,heads,groups,dim,vdim,rot", [(2, 9, 6, 2, 64, 32, 32), (1, 1, 4, 1, 128, 128, 128), (3, 5, 5, 5, 9, 11, 6),
                                                               (2, 3, 3, 1, 40, 7, 0), (1, 7, 2, 1, 320, 24, 320)])
def test_qkv_prep(dtype, batch, s, heads, groups, dim, vdim, rot):
    from oslo_b200.ops import cuda_ops
    n, past, tmax = batch * s, 4, s + 9
    p = rnd(n, heads * dim + groups * (dim + vdim) + 8, dtype=dtype)
    q, k, v = p[:, :heads * dim], p[:, heads * dim:(heads + groups) * dim], p[:, (heads + groups) * dim:(heads + groups) * dim + groups * vdim]
    wq, wk = rnd(dim, dtype=dtype), rnd(dim, dtype=dtype, seed=1)
    pos = torch.stack([torch.arange(past, past + s) + 1000 * b for b in range(batch)]).cuda()
    freq = torch.tensor(ref.rotary_frequencies(rot, 5e5), device="cuda")
    kc, vc = torch.zeros(batch, groups, tmax, dim, dtype=dtype, device="cuda"), torch.zeros(batch, groups, tmax, vdim, dtype=dtype, device="cuda")
    lengths = torch.full((batch,), past, dtype=torch.int32, device="cuda")
    got = cuda_ops.qkv_prep(q, k, v, wq, wk, 1e-4, pos, freq, kc, vc, lengths)
    close(got, ref.norm_rotate(q.reshape(batch, s, heads, dim), wq, 1e-4, pos, freq), dtype)
    close(kc[:, :, past:past + s].transpose(1, 2), ref.norm_rotate(k.reshape(batch, s, groups, dim), wk, 1e-4, pos, freq), dtype)
    assert torch.equal(vc[:, :, past:past + s].transpose(1, 2), v.reshape(batch, s, groups, vdim))
    for t in (kc, vc):
        t[:, :, past:past + s] = 0
        assert not t.any()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("batch,sq,sk,heads,groups,dim,vdim", [
    (2, 50, 50, 4, 1, 64, 64), (1, 2, 9, 4, 2, 24, 16), (2, 33, 70, 6, 3, 48, 80), (1, 140, 300, 4, 2, 128, 128), (1, 19, 19, 2, 1, 300, 20),
    (2, 130, 130, 4, 2, 192, 128), (1, 37, 37, 5, 1, 9, 11), (2, 200, 257, 8, 2, 64, 32), (1, 257, 257, 2, 2, 32, 136)])
def test_grouped_capped_attention(dtype, batch, sq, sk, heads, groups, dim, vdim):
    q, k, v = (rnd(batch, n, h, d, dtype=dtype, seed=i) for i, (n, h, d) in enumerate(((sq, heads, dim), (sk, groups, dim), (sk, groups, vdim))))
    k[:, 1] *= 6.0                                        # scores beyond the cap
    sink = torch.zeros(heads, dtype=dtype, device="cuda")
    keep = torch.ones(batch, sk, dtype=torch.uint8, device="cuda")
    keep[0, :min(7, sk - sq)] = 0
    for kp in (None, keep):
        for cap in (0.0, 2.0, 50.0):
            want, _ = ref.sink_attention(q, k, v, kp, sink, None, dim ** -0.5, cap)
            close(ops.sink_attention(q, k, v, kp, sink, None, dim ** -0.5, cap), want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("batch,heads,groups,dim,vdim,tmax,length", [
    (2, 6, 2, 64, 72, 200, 131), (1, 3, 1, 20, 12, 64, 1), (3, 17, 1, 48, 80, 96, 96), (1, 16, 4, 128, 128, 1500, 1400), (2, 8, 8, 32, 64, 300, 290),
    (9, 2, 1, 9, 11, 33, 20), (1, 40, 4, 64, 64, 700, 641), (2, 5, 5, 256, 256, 400, 390), (1, 4, 2, 16, 600, 50, 49), (40, 16, 2, 64, 32, 300, 257),
    (1, 8, 1, 320, 40, 300, 255)])
def test_grouped_decode(dtype, batch, heads, groups, dim, vdim, tmax, length):
    q = rnd(batch, heads, dim, dtype=dtype)
    k, v = rnd(batch, groups, tmax, dim, dtype=dtype), rnd(batch, groups, tmax, vdim, dtype=dtype, seed=2)
    k[:, :, 0] *= 5.0
    k[:, :, length:], v[:, :, length:] = float("nan"), float("nan")        # nothing beyond the valid length may be touched
    lengths = torch.full((batch,), length, dtype=torch.int32, device="cuda")
    lengths[0] = max(1, length - 3)
    sink = torch.zeros(heads, dtype=dtype, device="cuda")
    keep = torch.ones(batch, length, dtype=torch.uint8, device="cuda")
    keep[-1, :min(5, length - 1)] = 0
    from oslo_b200.ops import cuda_ops
    for kp in (None, keep):
        for cap in (0.0, 2.0, 50.0):
            want = ref.grouped_decode(q, torch.nan_to_num(k), torch.nan_to_num(v), lengths, kp, sink, dim ** -0.5, cap)
            close(cuda_ops.grouped_decode(q, k, v, lengths, kp, sink, dim ** -0.5, cap), want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_products_for_few_and_many_rows(dtype):
    for rows, k, n in ((1, 64, 40), (3, 128, 96), (9, 64, 48), (20, 64, 48), (70, 64, 24), (200, 72, 13), (5, 30, 9), (200, 64, 45), (70, 32, 434), (3, 64, 33)):
        x, w = rnd(4, rows, k, dtype=dtype), rnd(4, n, k, dtype=dtype, scale=k ** -0.5)
        close(torch.stack(ops.stacked_linear(x, w)), torch.matmul(x.float(), w.float().transpose(1, 2)), dtype)
        y = ops.linear_fp32(x[0], w[0])
        assert y.dtype == torch.float32
        close(y, x[0].float() @ w[0].float().t(), torch.float32)


def test_products_refuse_results_with_unaligned_rows():
    x, w = rnd(80, 64, dtype=torch.bfloat16), rnd(45, 64, dtype=torch.bfloat16)
    ext = ops.load_ext(required=True)
    with pytest.raises(RuntimeError, match="16-byte"):
        ext.gemm(x, w, 0, 0, None, None, None, None, 32, 1.0)          # 45 fp32 columns, rows without padding


# ---------------------------------------------------------------------------------------------------- the whole model
MODEL_TOL = {torch.float32: 5e-5, torch.bfloat16: 0.06}
WIDE = {
    # chunked recurrences and scans, several key tiles, cluster sizes above 1, more than one tile of query heads per key head
    "wide": case(200, 256, 1e-5, wkv(4, 64, dense(320), 32), mamba(512, 16, 16, 4, dense(192)),
                 parallel(attn(20, 2, 64, 64, 0.125, 20.0, 32), lin(4, 128, 64, (0.6, 0.9, 0.97, 0.999)), dense(256)),
                 mamba(384, 40, 24, 4, None), parallel(attn(4, 4, 128, 128, 0.1, 50.0, 128, 5e5), lin(8, 32, 96, [0.5 + 0.06 * i for i in range(8)]), None)),
}
ALL = {**{k: v for k, v in CASES.items() if k != "ones"}, **WIDE}


def load(tmp_path, cfg, tensors=None, dtype=torch.float32):
    tensors = make_tensors(cfg) if tensors is None else tensors
    write_model(str(tmp_path), cfg, tensors)
    model = ob.load_causal_lm(str(tmp_path), torch_dtype=dtype).cuda().fuse().eval()
    return model, tensors


def ids(n, vocab, seed=1):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def same(got, want, dtype, at=slice(None), factor=1.0):
    """Per position: root mean square over the vocabulary, relative to the logits' own."""
    got = got.double().cpu()
    assert torch.isfinite(got).all() and got.shape == want[at].shape
    d = (got - want[at]).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    assert float(d.max()) < factor * MODEL_TOL[dtype], float(d.max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", sorted(ALL))
def test_model_prompts_decoding_and_portions(tmp_path, dtype, name):
    cfg = ALL[name]
    model, tensors = load(tmp_path, cfg, dtype=dtype)
    n = 200 if name == "wide" else 70
    seq = ids(n, cfg["vocab"])
    want = plain.forward(cfg, tensors, seq)
    x = torch.tensor([seq], device="cuda")
    before = ops.load_ext(required=True).launch_count()
    with torch.no_grad():
        same(model(input_ids=x).logits[0], want, dtype)
        same(model(input_ids=x, use_cache=False).logits[0], want, dtype)
        assert ops.load_ext().launch_count() > before
        for portions in ([n - 12] + [1] * 12, [1] * 20, [2] * 6 + [n - 13, 1], [n // 2, 2, n - n // 2 - 2]):
            cache, at = StaticKVCache(16, grow=True), 0
            for m in portions:
                out = model(input_ids=x[:, at:at + m], past_key_values=cache, use_cache=True).logits[0]
                same(out, want, dtype, slice(at, at + m))
                at += m
    assert int(ops.load_ext().error_word(x).item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_model_batches_of_unequal_requests(tmp_path, dtype, name):
    cfg = ALL[name]
    model, tensors = load(tmp_path, cfg, dtype=dtype)
    lens, tails = (40, 1, 23, 150), (6, 9, 3, 2)
    seqs = [ids(a + b, cfg["vocab"], seed=a) for a, b in zip(lens, tails)]
    want = [plain.forward(cfg, tensors, s) for s in seqs]
    steps = BatchSteps(model, reserve=1)
    out = steps.start([s[:a] for s, a in zip(seqs, lens)])
    for r in range(4):
        same(out[r, steps.pad[r]:], want[r], dtype, slice(0, lens[r]))
    live, at = [0, 1, 2, 3], list(lens)
    while True:
        rows = [i for i, r in enumerate(live) if at[r] < len(seqs[r])]
        if not rows:
            break
        steps.keep(rows)
        live = [live[i] for i in rows]
        out = steps.advance([seqs[r][at[r]] for r in live])
        for i, r in enumerate(live):
            same(out[i, 0][None], want[r], dtype, slice(at[r], at[r] + 1))
            at[r] += 1


def test_model_many_rows_decode_like_few(tmp_path):
    cfg = WIDE["wide"]
    model, tensors = load(tmp_path, cfg, dtype=torch.bfloat16)
    seqs = [ids(30, 200, seed=s) for s in range(21)]
    want = [plain.forward(cfg, tensors, s) for s in seqs[:3]]
    x = torch.tensor(seqs, device="cuda")
    cache = StaticKVCache(40)
    with torch.no_grad():
        model(input_ids=x[:, :26], past_key_values=cache)
        for t in range(26, 30):
            out = model(input_ids=x[:, t:t + 1], past_key_values=cache).logits
            for r in range(3):
                same(out[r], want[r], torch.bfloat16, slice(t, t + 1))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_model_far_keys_on_the_gpu(tmp_path, dtype):
    cfg = case(64, 64, 1e-5, parallel(attn(4, 2, 64, 64, 0.125, 30.0, 16, 1e6), lin(1, 16, 16, (0.5,)), None), mamba(32, 8, 4, 4, dense(48)))
    tensors = far_key_weights(0, make_tensors(cfg, 3), 2.0)
    seq = [t % 60 for t in ids(420, 60, 8)]
    for at in (0, 1, 127, 128, 255):
        seq[at] = 63
    want = plain.forward(cfg, tensors, seq)
    other = plain.forward(cfg, tensors, [62] + seq[1:])
    model, _ = load(tmp_path, cfg, tensors, dtype)
    x = torch.tensor([seq], device="cuda")
    factor = 2.0 if dtype == torch.float32 else 1.0
    with torch.no_grad():
        same(model(input_ids=x).logits[0], want, dtype, factor=factor)
        cache = StaticKVCache(420)
        model(input_ids=x[:, :400], past_key_values=cache)
        got = torch.cat([model(input_ids=x[:, t:t + 1], past_key_values=cache).logits[0] for t in range(400, 420)])
    same(got, want, dtype, slice(400, None), factor)
    moved = (other[400:] - want[400:]).pow(2).mean(-1).sqrt().max() / want.pow(2).mean().sqrt()
    assert float(moved) > 20 * MODEL_TOL[torch.float32]   # the first token is seen from the end


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
    half, _ = load(tmp_path, cfg, tensors, dtype=torch.bfloat16)
    assert torch.equal(half.generate(x, **kw), half.generate(x, cuda_graph=True, **kw))


def test_model_with_sizes_beyond_one_kernel(tmp_path):
    cfg = case(40, 32, 1e-5, wkv(1, 300, None, 4), parallel(attn(2, 1, 300, 24, 0.06, 9.0, 300), lin(1, 700, 16, (0.9,)), None),
               mamba(16, 130, 3, 9, dense(24)))
    model, tensors = load(tmp_path, cfg)
    seq = ids(24, 40)
    want = plain.forward(cfg, tensors, seq)
    x = torch.tensor([seq], device="cuda")
    cache = StaticKVCache(24)
    with torch.no_grad():
        got = [model(input_ids=x[:, a:b], past_key_values=cache).logits[0] for a, b in ((0, 15), (15, 20), (20, 21), (21, 22))]
    same(torch.cat(got), want, torch.float32, slice(0, 22), 2.0)


def test_long_decoding_keeps_agreeing_with_the_prompt_form(tmp_path):
    cfg = CASES["heads64"]
    for dtype in (torch.float32, torch.bfloat16):
        model, tensors = load(tmp_path, cfg, dtype=dtype)
        seq = ids(400, 128, 5)
        want = plain.forward(cfg, tensors, seq)
        x = torch.tensor([seq], device="cuda")
        cache = StaticKVCache(400)
        with torch.no_grad():
            model(input_ids=x[:, :3], past_key_values=cache)
            got = torch.cat([model(input_ids=x[:, t:t + 1], past_key_values=cache).logits[0] for t in range(3, 400)])
        same(got, want, dtype, slice(3, None), 1.5)
