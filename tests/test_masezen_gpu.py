"""The kernels behind Masezen against the fp32 PyTorch statements of the same ops, over sizes that do and do not fit the
vector widths and tiles, and the whole model on the GPU against the plain implementation in ``plain_masezen.py``."""

import pytest
import torch

import oslo_b200 as ob
from oslo_b200 import ops
from oslo_b200.generation import BatchSteps, GraphedGreedyDecoder
from oslo_b200.models.common import StaticKVCache
from oslo_b200.ops import reference as ref
from oslo_b200.ops.reference import Branch

from . import plain_masezen as plain
from .masezen_cases import CASES, YARN, attn, case, dense, make_tensors, moe, steady, write_model

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
    """``keep`` ``[batch, s]`` with padding on the left of every row but the last (at least ``real`` real tokens)."""
    keep = torch.ones(batch, s, dtype=torch.uint8, device="cuda")
    for b in range(batch - 1):
        keep[b, :min(s - real, 3 + 14 * b)] = 0
    return keep


def no_device_error(like):
    assert int(ops.load_ext(required=True).error_word(like).item()) == 0


# ---------------------------------------------------------------------------------------------------- attention
# heads, key / value heads, head size: keys of 8 to 1200 columns, one to four value sub-tiles, groups of one to twelve heads
HEADS = [(4, 2, 64), (6, 3, 16), (1, 1, 8), (5, 5, 24), (8, 2, 128), (12, 1, 128), (6, 6, 200), (16, 4, 128), (3, 3, 256), (20, 10, 104), (32, 4, 32), (18, 6, 40)]
RAGGED = [(4, 2, 7), (3, 1, 33), (2, 2, 1), (6, 2, 12)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,groups,dim", HEADS + RAGGED)
def test_queries_of_mixed_heads_and_cache_append(dtype, heads, groups, dim):
    from oslo_b200.ops import cuda_ops
    for batch, s, past, rot, halves in ((2, 9, 0, dim // 2 * 2, True), (3, 1, 5, dim // 4 * 2, True), (1, 70, 2, 0, False), (2, 3, 1, dim // 2 * 2, False)):
        p = rnd(batch * s, (heads + groups) * dim + 3, dtype=dtype)
        q, k = p[:, :heads * dim], p[:, heads * dim:(heads + groups) * dim]
        wq, wk, talk = rnd(dim, dtype=dtype), rnd(dim, dtype=dtype, seed=1), rnd(heads, heads, dtype=dtype, seed=2)
        freq = torch.tensor(ref.rotary_frequencies(rot, 500.0, YARN), dtype=torch.float32, device="cuda")
        pos = torch.arange(past, past + s, device="cuda")[None].expand(batch, s) + torch.arange(batch, device="cuda")[:, None]
        lengths = torch.full((batch,), past, dtype=torch.int32, device="cuda")
        qh, kh = q.reshape(batch, s, heads, dim), k.reshape(batch, s, groups, dim)
        for mix in (talk, None):
            if mix is None:
                ks, vs = (torch.zeros(batch, groups, past + s + 2, dim, dtype=dtype, device="cuda") for _ in range(2))
            else:
                ks, vs = (torch.zeros(batch, past + s + 2, groups, dim, dtype=dtype, device="cuda").transpose(1, 2) for _ in range(2))
            for weights in ((wq, wk), (None, None)):
                got = cuda_ops.head_prep(q, k, k, *weights, 1e-3, pos, freq, halves, 1.1, mix, ks, vs, lengths)
                if mix is None:
                    want = ref.norm_rotate(qh, weights[0], 1e-3, pos, freq, halves, 1.1)
                else:
                    want = ref.norm_rotate_fold(qh, weights[0], 1e-3, pos, freq, mix, groups, halves, 1.1)
                close(got, want, dtype)
                close(ks[:, :, past:past + s].transpose(1, 2), ref.norm_rotate(kh, weights[1], 1e-3, pos, freq, halves, 1.1), dtype)
                assert torch.equal(vs[:, :, past:past + s].transpose(1, 2), kh)
                assert not ks[:, :, :past].any() and not ks[:, :, past + s:].any() and not vs[:, :, past + s:].any()
        # a position outside the cache is never written
        before = ks.clone()
        cuda_ops.head_prep(q, k, k, wq, wk, 1e-3, pos, freq, halves, 1.1, None, ks, vs, lengths + 1000)
        assert torch.equal(ks, before)
    ops.load_ext().error_word(p).zero_()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,groups,dim", HEADS + RAGGED)
def test_prompt_attention_with_wide_keys(dtype, heads, groups, dim):
    wide = groups * dim
    sizes = ((2, 130, 130), (1, 5, 300), (3, 257, 260)) if dtype != torch.float32 else ((2, 40, 40), (1, 5, 75))
    for batch, sq, sk in sizes:
        q = rnd(batch, sq, heads, wide, dtype=dtype, scale=2.0 * wide ** -0.25)
        k, v = rnd(batch, sk, wide, dtype=dtype, scale=wide ** -0.25), rnd(batch, sk, groups, dim, dtype=dtype)
        gate, narrow = rnd(batch * sq, heads * dim, dtype=dtype, scale=2.0), rnd(batch * sq, heads, dtype=dtype, scale=2.0)
        keep = padding(batch, sk, sk - sq + 1 if sk > sq else 1)
        for kp, g in ((None, gate), (keep, None), (keep, gate), (None, narrow)):
            got = ops.sink_attention(q, k[:, :, None], v, kp, None, g, 0.7)
            want = ref.sink_attention(q, k[:, :, None], v, kp, None, g, 0.7)[0]
            close(got, want, dtype)
        lead = (keep.cumsum(-1) == 0).sum(-1, dtype=torch.int32)
        sink = rnd(heads, dtype=dtype)
        close(ops.sink_attention(q, k[:, :, None], v, keep, sink, gate, 0.7, 0.0, 20, 3, lead),
              ref.sink_attention(q, k[:, :, None], v, keep, sink, gate, 0.7, 0.0, 20, 3, lead)[0], dtype)
    no_device_error(q)


def test_prompt_attention_finds_one_key_among_many():
    """A single score stands out, at block borders and far away; every query sees it from its place on and none before."""
    heads, groups, dim, n = 4, 2, 64, 700
    for at in (0, 1, 127, 128, 255, 256, 511, 640):
        q, k = torch.zeros(1, n, heads, groups * dim, device="cuda"), torch.zeros(1, n, 1, groups * dim, device="cuda")
        q[..., 5], k[:, at, 0, 5] = 8.0, 8.0
        v = torch.zeros(1, n, groups, dim, device="cuda")
        v[:, at] = 1.0
        o = ops.sink_attention(*(t.to(torch.bfloat16) for t in (q, k, v)), None, None, None, 1.0).view(n, -1).float()
        assert float(o[at:].min()) > 0.99 and not o[:at].any(), at


def test_prompt_attention_is_the_same_every_time():
    """Bit for bit, with operands in L2 and not: the roles of a block meet in whatever order loads arrive."""
    ext, other = ops.load_ext(required=True), torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    for b, s, t, h, g, d in ((3, 257, 260, 20, 10, 104), (2, 300, 300, 16, 4, 128)):
        q = rnd(b, h, s, g * d, dtype=torch.bfloat16, scale=2.0 * (g * d) ** -0.25)
        k, v = rnd(b, 1, t, g * d, dtype=torch.bfloat16, scale=(g * d) ** -0.25), rnd(b, g, t, d, dtype=torch.bfloat16)
        kq, kk = rnd(b, h, s, 128, dtype=torch.bfloat16), rnd(b, g, t, 128, dtype=torch.bfloat16)
        for run in (lambda: ext.flash_wide_fwd(q, k, v, None, None, None, 0.7), lambda: ext.flash_sink_fwd(kq, kk, v, None, None, None, 0.2, 0.0)):
            first = run()
            for i in range(20):
                if i % 2:
                    other.zero_()
                assert torch.equal(run(), first), i


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,groups,dim", HEADS + RAGGED)
def test_decode_attention_with_wide_keys(dtype, heads, groups, dim):
    from oslo_b200.ops import cuda_ops
    wide, room = groups * dim, 290
    for batch, lens in ((1, (1,)), (3, (290, 17, 129)), (9, (33, 32, 31, 16, 64, 65, 200, 289, 2))):
        q = rnd(batch, heads, wide, dtype=dtype, scale=2.0 * wide ** -0.25)
        ks, vs = rnd(batch, 1, room, wide, dtype=dtype, scale=wide ** -0.25), rnd(batch, 1, room, wide, dtype=dtype, seed=3)
        v = vs.view(batch, room, groups, dim).transpose(1, 2)
        lengths = torch.tensor(lens, dtype=torch.int32, device="cuda")
        gate, narrow = rnd(batch, heads * dim, dtype=dtype, scale=2.0), rnd(batch, heads, dtype=dtype, scale=2.0)
        keep = torch.ones(batch, room - 3, dtype=torch.uint8, device="cuda")
        keep[0, :min(lens) // 2] = 0
        for kp, g in ((None, gate), (keep, gate), (keep, None), (None, narrow)):
            got = cuda_ops.grouped_decode(q, ks, v, lengths, kp, None, 0.7, 0.0, g)
            close(got, ref.grouped_decode(q, ks, v, lengths, kp, None, 0.7, 0.0, g), dtype)
        lead, sink = torch.full((batch,), min(lens) // 2, dtype=torch.int32, device="cuda"), rnd(heads, dtype=dtype)
        keep[:, :min(lens) // 2] = 0
        close(cuda_ops.grouped_decode(q, ks, v, lengths, keep, sink, 0.7, 0.0, gate, 12, 4, lead),
              ref.grouped_decode(q, ks, v, lengths, keep, sink, 0.7, 0.0, gate, 12, 4, lead), dtype)
    # what lies past a sequence's end has no influence, whatever it is
    ks[:, :, lens[0]:], vs[:, :, lens[0]:] = 1e4, float("inf")
    one = slice(0, 1)
    close(cuda_ops.grouped_decode(q[one], ks[one], v[one], lengths[one], None, None, 0.7, 0.0, gate[one]),
          ref.grouped_decode(q[one], ks[one], v[one], lengths[one], None, None, 0.7, 0.0, gate[one]), dtype)
    no_device_error(q)


# ---------------------------------------------------------------------------------------------------- convolution, joins, token input
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [64, 36, 33, 300])
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 9])
def test_input_convolution(dtype, width, taps):
    for batch, s in ((1, 1), (2, 7), (3, 100), (2, 16), (1, 17)):
        x, w = rnd(batch * s, width, dtype=dtype), rnd(width, taps, dtype=dtype)
        prev = rnd(batch, taps - 1, width)
        for keep in (None, padding(batch, s)):
            want, last = ref.causal_conv(x, w, None, batch, keep, prev, residual=True)
            state = prev.clone()
            close(ops.causal_conv(x, w, None, batch, keep, state, residual=True), want, dtype)
            assert torch.equal(state, last)
            close(ops.causal_conv(x, w, None, batch, keep, None), ref.causal_conv(x, w, None, batch, keep, None)[0], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width", [(1, 64), (3, 2048), (70, 1027), (5, 33), (300, 1280), (2, 4100)])
def test_joins(dtype, rows, width):
    from oslo_b200.ops import cuda_ops
    x, ls, w = rnd(rows, width), rnd(width, dtype=dtype), rnd(width, dtype=dtype, seed=1)
    a, b, c = (rnd(rows, width, dtype=dtype, seed=i) for i in (2, 3, 4))
    top = 3
    many = rnd(rows * top + 11, width, dtype=dtype, seed=5)
    slots = torch.randperm(rows * top + 11, generator=torch.Generator().manual_seed(rows))[:rows * top].view(rows, top).to(torch.int32).cuda()
    lists = ([Branch(a, ls, normed=False), Branch(many, ls, 0.5, False, slots, top), Branch(c, w, normed=False)],
             [Branch(a, ls, normed=False), Branch(many[:rows * top], w, normed=False, top=top)], [Branch(a, w), Branch(many, w, 1.0, True, slots, top)], [Branch(b)])
    one = torch.tensor(0.8, dtype=dtype, device="cuda")
    for branches in lists:
        want, (copy,) = ref.branch_join(x, branches, 0.7, 1e-5, [], copy=dtype)
        got, (mine,) = ops.branch_join(x, branches, 0.7, 1e-5, [], copy=dtype)
        close(got, want, torch.float32)
        assert torch.equal(mine, got.to(dtype))
        for norms in ([one], [w], [one, w], [w, one]):
            got, hs = ops.branch_join(x, branches, 0.7, 1e-5, norms)
            _, want_h = ref.branch_join(x, branches, 0.7, 1e-5, norms)
            for h, wh in zip(hs, want_h):
                close(h, wh, dtype)
    close(ops.rms_norm(x, one, 1e-5), ref.rms_norm(x, one, 1e-5), dtype)
    for taps in (1, 2, 4, 6):
        cw, prev = rnd(width, taps, dtype=dtype), rnd(rows, taps - 1, width)
        for keep in (None, padding(rows, 1, 0)):
            state = prev.clone()
            got, (h, conv) = cuda_ops.branch_join(x, [Branch(a, w)], 1.0, 1e-5, [one], None, (cw, state, keep))
            want, last = ref.causal_conv(h, cw, None, rows, keep, prev, residual=True)
            close(conv, want, dtype)
            assert torch.equal(state, last)
            none = cuda_ops.branch_join(x, [Branch(a, w)], 1.0, 1e-5, [one], None, (cw, None, keep))[1][1]
            close(none, ref.causal_conv(h, cw, None, rows, keep, None, residual=True)[0], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,dim,first", [(1, 24, 48), (300, 64, 64), (5, 7, 3), (2, 256, 0)])
def test_token_gate(dtype, rows, dim, first):
    z, table = rnd(rows, dim + 8, dtype=dtype, scale=3.0)[:, :dim], rnd(50, first + dim + 4, dtype=dtype)
    tokens = torch.randint(0, 50, (rows, 2), generator=torch.Generator().manual_seed(1)).cuda()[:, 1]
    close(ops.token_gate(z, tokens, table, first), ref.token_gate(z, tokens, table, first), dtype)


# ---------------------------------------------------------------------------------------------------- feed-forward
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 3, 7, 64, 200])
@pytest.mark.parametrize("width,ff", [(64, 96), (256, 1024), (35, 21)])
def test_squared_relu_products(dtype, rows, width, ff):
    x, w = rnd(rows, width, dtype=dtype), rnd(ff, width, dtype=dtype, scale=width ** -0.5)
    with torch.no_grad():
        close(ops.linear(x, w, None, False, "relu2"), torch.relu(x.float() @ w.float().t()).pow(2), dtype, 2.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width,outputs,top", [(1, 256, 20, 4), (7, 100, 6, 6), (64, 37, 5, 1), (65, 64, 33, 8), (300, 128, 300, 5), (90, 64, 1, 1)])
def test_sigmoid_routing(dtype, rows, width, outputs, top):
    h, w = rnd(rows, width, dtype=dtype), rnd(outputs, width, dtype=dtype, scale=2.0 * width ** -0.5)
    idx, weights = ops.moe_route(h, w, None, top, "sigmoid")
    want_idx, want = ref.moe_route(h, w, None, top, "sigmoid")
    z = h.float() @ w.float().t()
    assert torch.allclose(z.gather(1, idx.long()), z.gather(1, want_idx.long()), atol=1e-4)   # equal choices up to close calls
    assert all(len(set(r)) == top for r in idx.tolist())
    same = (idx == want_idx).all(1)
    assert same.float().mean() > 0.9
    close(weights[same], want[same], torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width,ff,experts,top", [(1, 64, 24, 4, 3), (2, 48, 96, 6, 4), (40, 64, 40, 5, 4), (300, 128, 64, 8, 3), (33, 35, 13, 3, 2), (2, 35, 7, 5, 4),
                                                       (70, 256, 256, 2, 2), (50, 40, 136, 3, 1)])
def test_clamped_experts_with_scaled_inputs(dtype, rows, width, ff, experts, top):
    g = torch.Generator().manual_seed(rows)
    h, up, down = rnd(rows, width, dtype=dtype), rnd(experts, 2 * ff, width, dtype=dtype, scale=2.0 * width ** -0.5), rnd(experts, width, ff, dtype=dtype, scale=ff ** -0.5)
    idx = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(rows)]).to(torch.int32).cuda()
    weights = torch.rand(rows, top, generator=g).cuda()
    for limit, alpha, scale in ((0.7, 1.702, weights), (5.0, 0.9, weights), (0.7, 1.702, None)):
        y, slots = ops.moe_experts(h, idx, up, down, "clamped", limit, alpha, scale)
        want = ref.moe_experts(h, idx, up, down, "clamped", limit, alpha, scale).view(rows, top, width)
        at = torch.arange(rows * top, device="cuda").view(rows, top) if slots is None else slots.long()
        close(y[at], want, dtype)


# ---------------------------------------------------------------------------------------------------- the whole model
MODEL_TOL = 1e-4   # 32-bit
BIG = {"factor": 4.0, "original": 64, "fast": 16.0, "slow": 1.0}
WIDE = {
    # several key tiles, resident and streamed queries, more than one tile of heads, routed batches, a dense product on CTA pairs' rows
    "wide": case(200, 272, 1e-6, 4, 40, attn(20, 10, 64, 0.12, 32, moe(88, 18, 3, 2.0, 136, 1.0), 1e4, BIG), attn(8, 2, 128, 0.1, 128, dense(512), 5e5),
                 attn(36, 4, 32, 0.17, 32, moe(64, 8, 2, 1.0), 1e4, BIG), attn(4, 4, 128, 0.08, 96, None, 1e5, YARN)),
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
    n = 150 if name == "wide" else 70
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
    no_device_error(x)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_model_batches_of_unequal_requests(tmp_path, dtype, name):
    cfg = ALL[name]
    model, tensors = load(tmp_path, cfg, dtype=dtype)
    lens, tails = (40, 1, 23, 131), (6, 9, 3, 2)
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
    seqs = [ids(34, 200, seed=s) for s in range(70)]
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
def test_model_far_keys_and_first_tokens(tmp_path, dtype):
    cfg = case(64, 64, 1e-6, 4, 16, attn(4, 2, 64, 0.3, 16, None, 1e6, BIG), attn(2, 2, 16, 0.3, 8, dense(32)))
    tensors = make_tensors(cfg, 3)
    for name in ("l0.mix.q.norm", "l0.mix.k.norm"):
        tensors[name] = tensors[name] * 1.3
    seq = [t % 60 for t in ids(320, 60, 8)]
    for at in (0, 1, 127, 128, 255):
        seq[at] = 63
    want = Want(cfg, tensors, seq, dtype)
    other = plain.forward(cfg, tensors, [62] + seq[1:])
    model, _ = load(tmp_path, cfg, tensors, dtype)
    same(model(input_ids=torch.tensor([seq], device="cuda")).logits[0].detach(), want, dtype, factor=2.0)
    same(fed(model, seq, 300), want, dtype, factor=2.0)
    moved = (other[300:] - want.logits[300:]).pow(2).mean(-1).sqrt().max() / want.logits.pow(2).mean().sqrt()
    assert float(moved) > 10 * MODEL_TOL   # the first token is seen from the end


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
    for _ in range(2):                                    # the captured step (its two branches), the cache and the states are used again
        assert torch.equal(dec.generate(x, 10).cpu(), want)
    assert dec.replays > 0
    # the 16-bit model decodes the same tokens eagerly and from the captured step
    half, _ = load(tmp_path, cfg, dtype=torch.bfloat16)
    assert torch.equal(half.generate(x, **kw), half.generate(x, cuda_graph=True, **kw))


def test_model_with_sizes_beyond_one_kernel(tmp_path):
    """Keys and values wider than the decode kernels' shared memory, more heads than a block takes."""
    cfg = case(40, 32, 1e-5, 11, 8, attn(6, 6, 264, 0.06, 264, moe(8, 70, 66, 1.0, 16)), attn(34, 34, 64, 0.1, 64, None))
    for dtype in (torch.float32, torch.bfloat16):
        model, tensors = load(tmp_path, cfg, dtype=dtype)
        seq = ids(24, 40)
        want = Want(cfg, tensors, seq, dtype)
        x = torch.tensor([seq], device="cuda")
        cache = StaticKVCache(24)
        with torch.no_grad():
            got = [model(input_ids=x[:, a:b], past_key_values=cache).logits[0] for a, b in ((0, 15), (15, 20), (20, 21), (21, 22))]
        same(torch.cat(got), want, dtype, slice(0, 22), 2.0)


def test_long_decoding_keeps_agreeing_with_the_prompt_form(tmp_path):
    cfg = CASES["heads64"]
    for dtype in (torch.float32, torch.bfloat16):
        model, tensors = load(tmp_path, cfg, dtype=dtype)
        seq = ids(200, 128, 5)
        want = Want(cfg, tensors, seq, dtype)
        same(fed(model, seq, 3), want, dtype, factor=1.5)
