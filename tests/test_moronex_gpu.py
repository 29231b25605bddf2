"""The kernels behind Moronex against the fp32 PyTorch statements of the same ops, over sizes that do and do not fit the
vector widths and tiles, and the whole model on the GPU against the plain implementation in ``plain_moronex.py``."""
import pytest
import torch

import oslo_b200 as ob
from oslo_b200 import ops
from oslo_b200.generation import BatchSteps, GraphedGreedyDecoder
from oslo_b200.models.common import StaticKVCache
from oslo_b200.ops import reference as ref

from . import plain_moronex as plain
from .moronex_cases import CASES, case, dense, far_key_weights, hgrn2, latent, make_tensors, moe, write_model

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
@pytest.mark.parametrize("batch,s,heads,dim,vdim", [(2, 37, 3, 40, 72), (1, 1, 2, 16, 8), (1, 200, 1, 12, 20), (2, 17, 2, 100, 33),
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
@pytest.mark.parametrize("batch,heads,dim,vdim", [(1, 5, 40, 72), (5, 3, 20, 30), (2, 16, 128, 128), (70, 2, 64, 256), (1, 1, 7, 2100)])
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
@pytest.mark.parametrize("batch,heads,dim,vdim,rank,tmax,length", [(2, 6, 64, 72, 112, 200, 131), (1, 3, 20, 12, 40, 64, 1),
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
        got, _ = cuda_ops.latent_prep(p[:, 8:136], wq, p[:, 200:272], wk, cache, lengths, 1e-5)
        close(got, ref.rms_norm(p[:, 8:136], wq, 1e-5), dtype)
        close(cache[:, 4], ref.rms_norm(p[:, 200:272], wk, 1e-5), dtype)
        cache[:, 4] = 0
        assert not cache.any()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,width,ff,experts,top", [(1, 64, 32, 4, 2), (5, 40, 24, 3, 3), (4, 192, 104, 9, 2), (17, 192, 104, 9, 2),
                                                       (200, 128, 300, 5, 1), (300, 36, 20, 7, 3), (700, 512, 256, 16, 4), (300, 64, 24, 37, 3)])
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


# ---------------------------------------------------------------------------------------------------- the whole model
MODEL_TOL = {torch.float32: 5e-5, torch.bfloat16: 0.08}
WIDE = {
    # chunked recurrences, several key tiles, the grouped expert product, cluster sizes above 1
    "wide": case(200, 256, 1e-5, hgrn2(4, 128, 64, moe(128, 6, 2)), latent(6, 64, 64, 128, 128, 0.125, moe(96, 4, 3)),
                 latent(18, 32, 48, 96, 128, 0.2, dense(320), kv_from=1), hgrn2(2, 24, 136, None)),
}
ALL = {**CASES, **WIDE}


def load(tmp_path, cfg, tensors=None, dtype=torch.float32):
    tensors = make_tensors(cfg) if tensors is None else tensors
    write_model(str(tmp_path), cfg, tensors)
    model = ob.load_causal_lm(str(tmp_path), torch_dtype=dtype).cuda().fuse().eval()
    return model, tensors


def ids(n, vocab, seed=1):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


class Want:
    """The plain model's logits of a sequence, and the positions that 16-bit rounding does not blow up (a router's close call, a
    post-norm of next to nothing): those where weights off by a fraction of a 16-bit step change little."""

    def __init__(self, cfg, tensors, seq):
        self.logits = plain.forward(cfg, tensors, seq)
        g = torch.Generator().manual_seed(77)
        self.clear = torch.ones(len(seq), dtype=torch.bool)
        for _ in range(2):
            off = {k: t.double() * (1 + 2.0 ** -9 * torch.randn(t.shape, generator=g)) for k, t in tensors.items()}
            d = (plain.forward(cfg, off, seq) - self.logits).pow(2).mean(-1).sqrt() / self.logits.pow(2).mean().sqrt()
            self.clear &= d < 0.03
        assert self.clear.double().mean() > 0.5


def errors(got, want, dtype, at=slice(None)):
    """Per position: root mean square over the vocabulary, relative to the logits' own."""
    ref_rows, clear = want.logits[at], want.clear[at]
    got = got.double().cpu()
    assert torch.isfinite(got).all() and got.shape == ref_rows.shape
    d = (got - ref_rows).pow(2).mean(-1).sqrt() / want.logits.pow(2).mean().sqrt()
    return d if dtype == torch.float32 else d[clear]


def small(d, dtype, factor=1.0):
    """In 32-bit every position counts; in 16-bit one position in thirty may be one that rounding blows up all the same."""
    over = int((d > factor * MODEL_TOL[dtype]).sum())
    assert over <= (0 if dtype == torch.float32 else -(-d.numel() // 30)), (over, d.numel(), float(d.max()))


def same(got, want, dtype, at=slice(None), factor=1.0):
    small(errors(got, want, dtype, at), dtype, factor)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", sorted(ALL))
def test_model_prompts_decoding_and_portions(tmp_path, dtype, name):
    cfg = ALL[name]
    model, tensors = load(tmp_path, cfg, dtype=dtype)
    n = 150 if name == "wide" else 70
    seq = ids(n, cfg["vocab"])
    want = Want(cfg, tensors, seq)
    x = torch.tensor([seq], device="cuda")
    before = ops.load_ext(required=True).launch_count()
    with torch.no_grad():
        same(model(input_ids=x).logits[0], want, dtype)
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
    lens, tails = (40, 1, 23, 70), (6, 9, 3, 2)
    seqs = [ids(a + b, cfg["vocab"], seed=a) for a, b in zip(lens, tails)]
    want = [Want(cfg, tensors, s) for s in seqs]
    steps = BatchSteps(model, reserve=1)
    out = steps.start([s[:a] for s, a in zip(seqs, lens)])
    for r in range(4):
        same(out[r, steps.pad[r]:], want[r], dtype, slice(0, lens[r]))
    live, at, d = [0, 1, 2, 3], list(lens), []
    while True:
        rows = [i for i, r in enumerate(live) if at[r] < len(seqs[r])]
        if not rows:
            break
        steps.keep(rows)
        live = [live[i] for i in rows]
        out = steps.advance([seqs[r][at[r]] for r in live])
        for i, r in enumerate(live):
            d.append(errors(out[i, 0][None], want[r], dtype, slice(at[r], at[r] + 1)))
            at[r] += 1
    small(torch.cat(d), dtype, 1.5)


def test_model_many_rows_decode_like_few(tmp_path):
    """The decode kernels for batches (tensor-core projections, grouped experts) against one row at a time."""
    cfg = WIDE["wide"]
    model, tensors = load(tmp_path, cfg, dtype=torch.bfloat16)
    seqs = [ids(30, 200, seed=s) for s in range(21)]
    want = [Want(cfg, tensors, s) for s in seqs[:3]]
    x = torch.tensor(seqs, device="cuda")
    cache, d = StaticKVCache(40), []
    with torch.no_grad():
        model(input_ids=x[:, :26], past_key_values=cache)
        for t in range(26, 30):
            out = model(input_ids=x[:, t:t + 1], past_key_values=cache).logits
            for r in range(3):
                d.append(errors(out[r], want[r], torch.bfloat16, slice(t, t + 1)))
    small(torch.cat(d), torch.bfloat16, 1.5)


def test_model_far_keys_on_the_gpu(tmp_path):
    cfg = case(64, 64, 1e-5, latent(2, 64, 64, 64, 64, 1.0, None), latent(3, 32, 64, 64, 64, 1.0, None, kv_from=0),
               hgrn2(2, 16, 32, dense(48)))
    tensors = far_key_weights(cfg, 0, make_tensors(cfg, 3))
    seq = [t % 60 for t in ids(420, 60, 8)]
    for at in (0, 1, 127, 128, 255):
        seq[at] = 63
    want = Want(cfg, tensors, seq)
    other = plain.forward(cfg, tensors, [62] + seq[1:])
    model, _ = load(tmp_path, cfg, tensors)
    x = torch.tensor([seq], device="cuda")
    with torch.no_grad():
        same(model(input_ids=x).logits[0], want, torch.float32, factor=2.0)
        cache = StaticKVCache(420)
        model(input_ids=x[:, :400], past_key_values=cache)
        got = torch.cat([model(input_ids=x[:, t:t + 1], past_key_values=cache).logits[0] for t in range(400, 420)])
    same(got, want, torch.float32, slice(400, None), 2.0)
    moved = (other[400:] - want.logits[400:]).pow(2).mean(-1).sqrt().max() / want.logits.pow(2).mean().sqrt()
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


def test_model_with_heads_and_latents_beyond_one_kernel(tmp_path):
    cfg = case(40, 32, 1e-5, hgrn2(1, 700, 16, None), latent(2, 20, 300, 24, 1100, 0.2, None))
    model, tensors = load(tmp_path, cfg)
    seq = ids(24, 40)
    want = Want(cfg, tensors, seq)
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
        want = Want(cfg, tensors, seq)
        x = torch.tensor([seq], device="cuda")
        cache = StaticKVCache(400)
        with torch.no_grad():
            model(input_ids=x[:, :3], past_key_values=cache)
            got = torch.cat([model(input_ids=x[:, t:t + 1], past_key_values=cache).logits[0] for t in range(3, 400)])
        same(got, want, dtype, slice(3, None), 1.5)
