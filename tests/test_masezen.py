"""Masezen on the CPU statements of the ops: every mechanism against ``plain_masezen.py`` (double precision, loops), the cache and the
convolution states under decoding, portions, padded batches, reordering and reuse, the scheduler and sampling paths of
``generate()``, loading, and the trace runner."""
import json
import math
import os
import subprocess

import pytest
import torch

import oslo_b200 as ob
from oslo_b200 import ops
from oslo_b200.generation import BatchSteps, GraphedGreedyDecoder
from oslo_b200.models.common import StaticKVCache
from oslo_b200.models.mixers import DenseMLP, GroupedQueryAttention, InputConvolution, MixtureOfExperts, TokenInput
from oslo_b200.ops.reference import Branch
from oslo_b200.parallel.layers import RMSNorm

from . import plain_masezen as plain
from .masezen_cases import CASES, YARN, attn, case, dense, make_tensors, moe, write_model

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = 5e-5


def load(tmp_path, cfg, tensors=None, seed=0, dtype=torch.float32):
    tensors = make_tensors(cfg, seed) if tensors is None else tensors
    write_model(str(tmp_path), cfg, tensors)
    return ob.load_causal_lm(str(tmp_path), torch_dtype=dtype).eval(), tensors


def ids(n, vocab, seed=1):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def err(a, b):
    a, b = a.detach().double(), b.detach().double()
    return float((a - b).abs().max() / b.abs().max().clamp(min=1e-6))


@torch.no_grad()
def logits(model, *seqs):
    return model(input_ids=torch.tensor(seqs)).logits


def randomise(module, std=0.5):
    for p in module.parameters():
        p.data.normal_(std=std)
    return module


def getter(table):
    table = {k: v.detach().double() for k, v in table.items()}
    return table.__getitem__


# ---------------------------------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("scaling", [None, YARN, {**YARN, "factor": 1.0}, {**YARN, "factor": 16.0, "fast": 1000.0, "slow": 1e-6},
                                     {"factor": 2.0, "original": 7, "fast": 1.0, "slow": 1.0}])
@pytest.mark.parametrize("dims,base", [(2, 10.0), (6, 500.0), (32, 1e4), (64, 5e5)])
def test_rotation_frequencies(dims, base, scaling):
    want, amplitude = plain.frequencies({"dims": dims, "base": base, "scaling": scaling})
    got = ops.reference.rotary_frequencies(dims, base, scaling)
    assert all(math.isclose(a, b, rel_tol=1e-12) for a, b in zip(got, want)) and len(got) == dims // 2
    assert math.isclose(ops.reference.rotary_amplitude(scaling), amplitude, rel_tol=1e-12)
    plain_f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is not None:                               # between the frequency itself and its factor-th part
        assert all(f / scaling["factor"] - 1e-15 <= g <= f + 1e-15 for g, f in zip(got, plain_f))


def test_yarn_keeps_fast_pairs_and_slows_slow_ones():
    scaling = {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}
    got = ops.reference.rotary_frequencies(128, 10000.0, scaling)
    f = [10000.0 ** (-2.0 * i / 128) for i in range(64)]
    turns = [4096 * x / (2 * math.pi) for x in f]
    assert all(g == x for g, x, t in zip(got, f, turns) if t > 33) and any(t > 33 for t in turns)
    assert all(math.isclose(g, x / 4.0) for g, x, t in zip(got, f, turns) if t < 0.9) and any(t < 0.9 for t in turns)
    assert math.isclose(ops.reference.rotary_amplitude(scaling), 0.1 * math.log(4.0) + 1.0)


@pytest.mark.parametrize("halves", [True, False])
def test_norm_and_rotation(halves):
    rot = {"dims": 6, "base": 30.0, "scaling": YARN}
    x, w, first = torch.randn(1, 9, 3, 10), torch.randn(10), 41
    freq = torch.tensor(ops.reference.rotary_frequencies(6, 30.0, YARN), dtype=torch.float32)
    got = ops.reference.norm_rotate(x, w, 1e-2, torch.arange(first, first + 9)[None], freq, halves, ops.reference.rotary_amplitude(YARN))
    y = plain.rms(x[0].double(), 1e-2) * w.double()
    if halves:
        want = plain.rotate(y, rot, first)
    else:                                                 # the same turns on neighbours
        order = [0, 2, 4, 1, 3, 5, 6, 7, 8, 9]
        want = torch.empty_like(y)
        want[:, :, order] = plain.rotate(y[:, :, order], rot, first)
    assert err(got[0], want) < TOL
    assert err(got[0, :, :, 6:], y[:, :, 6:]) < TOL       # the rest passes unchanged, without the amplitude


@pytest.mark.parametrize("heads,groups,dim", [(1, 1, 4), (4, 2, 6), (6, 1, 3), (3, 3, 5)])
def test_mixed_heads_are_one_product_with_wide_keys(heads, groups, dim):
    n, t = 5, 12
    q, k, v = torch.randn(n, heads, dim), torch.randn(t, groups, dim), torch.randn(t, groups, dim)
    talk = torch.randn(heads, heads)
    want = plain.mixed_attention(q.double(), k.double(), v.double(), 0.6, talk.double())
    norm = plain.rms(q.double(), 1e-9)                    # the fold norms its queries: undone by the sizes
    size = (q.double() / norm)[..., :1]
    ones = torch.ones(dim)
    folded = ops.reference.norm_rotate_fold(q[None], ones, 1e-9, torch.zeros(1, n, dtype=torch.long), None, talk, groups)
    assert folded.shape == (1, n, heads, groups * dim)
    again = plain.mixed_attention(norm, k.double(), v.double(), 0.6, talk.double())
    o, _ = ops.reference.sink_attention(folded, k.reshape(1, t, 1, -1), v[None], None, None, None, 0.6)
    assert err(o.view(n, heads, dim), again) < TOL
    if heads == 1:
        one, _ = ops.reference.sink_attention(folded * size[None], k.reshape(1, t, 1, -1), v[None], None, None, None, 0.6)
        assert err(one.view(n, heads, dim), want) < TOL
    # an identity leaves the heads alone
    alone = ops.reference.norm_rotate_fold(q[None], ones, 1e-9, torch.zeros(1, n, dtype=torch.long), None, torch.eye(heads), groups)
    a, _ = ops.reference.sink_attention(alone, k.reshape(1, t, 1, -1), v[None], None, None, None, 0.6)
    b, _ = ops.reference.sink_attention(ops.reference.norm_rotate(q[None], ones, 1e-9, None, None), k[None], v[None], None, None, None, 0.6)
    assert err(a, b) < TOL


@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_input_convolution(taps):
    n, width = 11, 6
    h, module = torch.randn(n, width), randomise(InputConvolution(width, taps))
    w = module.weight.detach()
    want = h.double() + plain.convolve(h.double(), w.double())
    with torch.no_grad():
        assert err(module(h, 1, 0, None, None), want) < TOL
        for portions in ([1] * n, [2] * 5 + [1], [3, 8], [10, 1]):
            cache, at, got = StaticKVCache(n), 0, []
            for m in portions:
                got.append(module(h[at:at + m], 1, 0, cache, None))
                at += m
            assert err(torch.cat(got), want) < TOL
            state = cache.state[(0, "inputs")][0]
            assert state.shape == (taps - 1, width) and torch.equal(state, h[n - taps + 1:] if taps > 1 else h[:0])
        # padding ahead counts as zeros
        keep = torch.tensor([[0] * 3 + [1] * n])
        got = module(torch.cat([torch.randn(3, width), h]), 1, 0, None, keep)
        assert err(got[3:], want) < TOL and not got[:3].any()
    assert err(plain.convolve(h.double()[4:], w.double(), torch.cat([torch.zeros(taps, width), h[:4]]).double()[5:5 + taps - 1]),
               plain.convolve(h.double(), w.double())[4:]) < 1e-12


def test_join_scales_sums_and_copies():
    n, width, top, eps = 5, 8, 3, 1e-2
    x, a, b, ls1, ls2, w = torch.randn(n, width), torch.randn(n, width), torch.randn(40, width), torch.randn(width), torch.randn(width), torch.randn(width)
    slots = torch.randperm(40)[:n * top].view(n, top).to(torch.int32)
    want = x.double() + ls1.double() * a.double() + 0.5 * ls2.double() * b.double()[slots.long()].sum(1)
    got, (copy,) = ops.branch_join(x, [Branch(a, ls1, normed=False), Branch(b, ls2, 0.5, False, slots, top)], 1.0, eps, [], copy=torch.bfloat16)
    assert err(got, want) < TOL and copy.dtype == torch.bfloat16 and torch.equal(copy, got.to(torch.bfloat16))
    got, _ = ops.branch_join(x, [Branch(b[:n * top], ls2, normed=False, top=top)], 1.0, eps, [], copy=torch.float32)
    assert err(got, x.double() + ls2.double() * b[:n * top].double().view(n, top, width).sum(1)) < TOL
    one, prev, cw = torch.tensor(0.7), torch.randn(n, 2, width), torch.randn(width, 3)
    state = prev.clone()
    got, (h, c) = ops.branch_join(x, [Branch(a, w)], 1.0, eps, [one], conv=(cw, state, None))
    want = x.double() + plain.rms(a.double(), eps) * w.double()
    normed = plain.rms(want, eps) * 0.7
    assert err(got, want) < TOL and err(h, normed) < TOL
    for r in range(n):
        assert err(c[r], normed[r] + plain.convolve(normed[r:r + 1], cw.double(), prev[r].double())[0]) < TOL
    assert torch.equal(state, torch.stack([prev[:, 1], h], dim=1))


def test_norm_with_one_number():
    norm = RMSNorm(None, 1e-2)
    assert norm.weight.shape == ()
    norm.weight.data.fill_(-1.3)
    x = torch.randn(4, 9)
    assert err(norm(x), plain.rms(x.double(), 1e-2) * -1.3) < TOL


def test_token_input():
    width, dim, vocab, n, eps = 12, 5, 7, 9, 1e-3
    module, table = randomise(TokenInput(width, dim, 2 * dim, eps)), torch.randn(vocab, 4 * dim)
    x, tokens = 2.0 * torch.randn(n, width), torch.randint(0, vocab, (n,))
    with torch.no_grad():
        b = module(x, tokens, table)
        got, _ = ops.branch_join(x, [b], 1.0, eps, [])
    want = plain.token_input(x.double(), table[tokens, 2 * dim:3 * dim].double(), *(t.weight.detach().double() for t in (module.gate, module.proj, module.norm)), eps)
    assert err(got - x, want) < TOL


@pytest.mark.parametrize("top", [1, 3, 5])
def test_experts_read_their_weight_and_are_summed_without(top):
    n, width, ff, experts, limit = 30, 9, 4, 5, 0.8
    h = 1.5 * torch.randn(n, width)
    for shared in (None, 7):
        m = randomise(MixtureOfExperts(width, ff, experts, top, unit="clamped", scored="sigmoid", limit=limit, scale_input=True, shared_gate=False,
                                       shared=shared, shared_limit=0.3))
        assert m.correction is None and m.router.bias is None
        with torch.no_grad():
            f = m(h)
        assert f.weights is None and f.choice is None and f.shared_gate is None
        got = f.y.view(n, top, width).sum(1) + (0.0 if shared is None else f.shared)
        table = {"router": m.router.weight}
        for e in range(experts):
            table.update({f"e{e}.gate": m.up[e, 0::2], f"e{e}.up": m.up[e, 1::2], f"e{e}.down": m.down[e]})
        mlp = moe(ff, experts, top, limit, shared, 0.3)
        if shared is not None:
            s = m.shared
            table.update({"shared.gate": s.in_proj.part("gate"), "shared.up": s.in_proj.part("up"), "shared.down": s.down.weight})
        assert err(got, plain.moe(h.double(), getter(table), mlp)) < TOL
    idx, weights = ops.moe_route(h, m.router.weight, None, top, "sigmoid")
    want_idx, want = plain.route(h.double(), m.router.weight.detach().double(), top)
    assert torch.equal(idx.long(), want_idx) and err(weights, want) < TOL
    # the weight belongs to the input: experts are not linear
    y = ops.moe_experts(h, idx, m.up, m.down, "clamped", limit, 1.702, weights)[0].view(n, top, width)
    z = ops.moe_experts(h, idx, m.up, m.down, "clamped", limit, 1.702)[0].view(n, top, width) * weights.unsqueeze(-1)
    assert err(y, z) > 0.01
    with pytest.raises(ValueError):
        MixtureOfExperts(width, 4, 2, 1, scored="softmax")


def test_dense_unit_and_mixer_alone():
    width, n, eps = 18, 21, 1e-3
    h, pos = torch.randn(n, width), torch.arange(n)[None]
    with torch.no_grad():
        d = randomise(DenseMLP(width, 11))
        assert err(d(h).y, plain.squared_relu_mlp(h.double(), d.up.weight.double(), d.down.weight.double())) < TOL
        m = attn(6, 2, 8, 0.4, 4, None, 100.0, YARN)["mixer"]
        kw = dict(rot_dims=4, rot_base=100.0, rot_scaling=YARN, halves=True, sink=False, value_is_key=True, gate="element", talk=True)
        a = randomise(GroupedQueryAttention(width, 6, 2, 8, 8, 0.4, eps, **kw))
        assert torch.equal(GroupedQueryAttention(width, 6, 2, 8, 8, 0.4, eps, **kw).talk, torch.eye(6))
        get = getter({**{s: a.in_proj.part(s) for s in "qkg"}, "q.norm": a.q_norm.weight, "k.norm": a.k_norm.weight, "talk": a.talk, "o": a.out_proj.weight})
        assert err(a(h, 1, 0, None, None, pos).y, plain.attention(h.double(), get, m, eps)) < TOL
        # without the mix: the module's heads alone
        b = GroupedQueryAttention(width, 6, 2, 8, 8, 0.4, eps, **{**kw, "talk": False})
        b.load_state_dict({k: v for k, v in a.state_dict().items() if k != "talk"})
        a.talk.copy_(torch.eye(6))
        assert err(a(h, 1, 0, None, None, pos).y, b(h, 1, 0, None, None, pos).y) < TOL
        # attention weights over the mixed scores sum to one, causally
        probs = a(h, 1, 0, None, None, pos, True).probs
        assert probs.shape == (1, 6, n, n) and err(probs.sum(-1), torch.ones(1, 6, n)) < 1e-5 and not probs.triu(1).any()
    with pytest.raises(ValueError):
        GroupedQueryAttention(width, 2, 1, 8, 8, 0.4, eps, gate="row")


# ---------------------------------------------------------------------------------------------------- the whole model
@pytest.mark.parametrize("name", sorted(CASES))
def test_logits_and_residual_stream(tmp_path, name):
    cfg = CASES[name]
    model, tensors = load(tmp_path, cfg)
    seq = ids(29, cfg["vocab"])
    want, stream = plain.forward(cfg, tensors, seq, keep_layers=True)
    with torch.no_grad():
        out = model(input_ids=torch.tensor([seq]), output_hidden_states=True)
    assert err(out.logits[0], want) < TOL
    for i in range(len(cfg["layers"])):
        assert out.hidden_states[i + 1].dtype == torch.float32 and err(out.hidden_states[i + 1][0], stream[i]) < TOL
    model.fuse()                                          # on the CPU the fused modules run the same statements
    assert err(logits(model, seq)[0], want) < TOL
    with torch.no_grad():
        out = model(input_ids=torch.tensor([seq]), use_cache=False, output_attentions=True)
    assert err(out.logits[0], want) < TOL and out.past_key_values is None and all(p is not None for p in out.attentions)


@pytest.mark.parametrize("name", ["mixed", "odd", "heads64"])
def test_sixteen_bit_model_keeps_stream_and_states_in_32_bit(tmp_path, name):
    cfg = CASES[name]
    model, tensors = load(tmp_path, cfg, dtype=torch.bfloat16)
    seq = ids(20, cfg["vocab"])
    with torch.no_grad():
        out = model(input_ids=torch.tensor([seq]), output_hidden_states=True)
    assert all(h.dtype == torch.float32 for h in out.hidden_states)
    assert all(s.dtype == torch.float32 for s in out.past_key_values.state.values())
    want = plain.forward(cfg, tensors, seq)
    d = (out.logits[0].double() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    assert float(d.median()) < 0.05                       # a close call of a router may go the other way at some positions


@pytest.mark.parametrize("name", sorted(CASES))
def test_prefill_equals_token_by_token_and_portions(tmp_path, name):
    cfg = CASES[name]
    model, _ = load(tmp_path, cfg)
    seq = ids(37, cfg["vocab"])
    want = logits(model, seq)[0]
    for portions in ([1] * 37, [30, 1, 1, 1, 1, 1, 1, 1], [2] * 18 + [1], [3, 16, 2, 16], [36, 1], [1, 36]):
        cache, got, at = StaticKVCache(8, grow=True), [], 0
        for n in portions:
            with torch.no_grad():
                out = model(input_ids=torch.tensor([seq[at:at + n]]), past_key_values=cache, use_cache=True)
            got.append(out.logits[0])
            at += n
        assert cache.length == 37 and err(torch.cat(got), want) < TOL
    # what is kept: wide keys and values per token, the last inputs of every layer's convolution
    n, taps = len(cfg["layers"]), cfg["canon"]["taps"]
    assert sorted(cache.k) == sorted(cache.v) == list(range(n)) and not cache.latent
    assert all(cache.k[i].shape[1:] == (1, cache.max_len, m["kv_heads"] * m["dim"]) for i, m in enumerate(l["mixer"] for l in cfg["layers"]))
    assert {k: tuple(v.shape) for k, v in cache.state.items()} == {(i, "inputs"): (1, taps - 1, cfg["width"]) for i in range(n)}


@pytest.mark.parametrize("name", ["mixed", "odd", "heads64"])
def test_batches_of_unequal_requests_match_each_alone(tmp_path, name):
    cfg = CASES[name]
    model, _ = load(tmp_path, cfg)
    seqs = [ids(n, cfg["vocab"], seed=n) for n in (44, 1, 23, 7)]
    prompt = [38, 1, 19, 2]                               # the rest is fed token by token; shorter requests end earlier
    seqs[1] = seqs[1] + ids(3, cfg["vocab"], seed=99)
    alone = [logits(model, s)[0] for s in seqs]
    steps = BatchSteps(model, reserve=2)
    out = steps.start([s[:n] for s, n in zip(seqs, prompt)])
    for r, (s, n) in enumerate(zip(seqs, prompt)):
        assert err(out[r, steps.pad[r]:], alone[r][:n]) < TOL
    live, at = [0, 1, 2, 3], list(prompt)
    while live:
        rows = [i for i, r in enumerate(live) if at[r] < len(seqs[r])]
        if not rows:
            break
        steps.keep(rows)
        live = [live[i] for i in rows]
        out = steps.advance([seqs[r][at[r]] for r in live])
        for i, r in enumerate(live):
            assert err(out[i, 0], alone[r][at[r]]) < TOL, (r, at[r])
            at[r] += 1
    assert at == [len(s) for s in seqs]


def test_rows_that_end_give_their_storage_back_and_leave_no_trace(tmp_path):
    cfg = CASES["mixed"]
    model, _ = load(tmp_path, cfg)
    a, b = ids(12, 96, 3), ids(15, 96, 4)
    want = logits(model, b)[0]
    steps = BatchSteps(model)
    steps.start([a, b[:10]])
    held = lambda c: sum(t.numel() for d in (c.k, c.v, c.state) for t in d.values())            # noqa: E731
    before = held(steps.kwargs["past_key_values"])
    steps.keep([1])
    assert held(steps.kwargs["past_key_values"]) * 2 == before
    for t in range(10, 15):
        assert err(steps.advance([b[t]])[0, 0], want[t]) < TOL
    # a cache that is emptied and used again behaves like a new one
    cache = StaticKVCache(40)
    for seq in (ids(20, 96, 5), ids(9, 96, 6), ids(20, 96, 7)):
        cache.reset()
        with torch.no_grad():
            first = model(input_ids=torch.tensor([seq[:5]]), past_key_values=cache).logits[0]
            rest = model(input_ids=torch.tensor([seq[5:]]), past_key_values=cache).logits[0]
        assert err(torch.cat([first, rest]), logits(model, seq)[0]) < TOL
    full = StaticKVCache(6)
    with torch.no_grad(), pytest.raises(RuntimeError, match="overflow"):
        model(input_ids=torch.tensor([a]), past_key_values=full)


def fed(model, seq, prompt):
    """Logits of ``seq`` when its first ``prompt`` tokens come at once and the others one by one."""
    cache = StaticKVCache(len(seq))
    with torch.no_grad():
        out = [model(input_ids=torch.tensor([seq[:prompt]]), past_key_values=cache).logits[0]]
        out += [model(input_ids=torch.tensor([[t]]), past_key_values=cache).logits[0] for t in seq[prompt:]]
    return torch.cat(out)


def test_a_convolution_reaches_taps_tokens_and_no_further(tmp_path):
    """A changed token moves what the mixer reads at its own place and the next ``taps - 1``, in prompts and in decoding."""
    taps, n = 5, 40
    cfg = case(64, 24, 1e-5, taps, 8, attn(2, 1, 8, 0.3, 4, None))
    tensors = make_tensors(cfg, 5)
    model, _ = load(tmp_path, cfg, tensors)
    block = model.transformer.h[0]
    seq = [t % 60 for t in ids(n, 60, 8)]
    seen = []
    hook = block.mixer.register_forward_hook(lambda m, args, out: seen.append(args[0].detach().clone()))

    def convolved(s, prompt):
        seen.clear()
        fed(model, s, prompt)
        return torch.cat(seen)

    for prompt in (n, 17, 2):
        base = convolved(seq, prompt)
        for at in (0, 1, taps - 1, 15, 16, 17, 18, n - 1):
            other = list(seq)
            other[at] = 61
            moved = (convolved(other, prompt) - base).abs().amax(-1)
            for i in range(n):
                assert (float(moved[i]) > 1e-3) == (at <= i < at + taps), (prompt, at, i)
    hook.remove()


def test_keys_far_away_and_first_tokens_decide_the_output(tmp_path):
    cfg = case(64, 40, 1e-5, 4, 8, attn(4, 2, 16, 0.5, 8, None, 1e5, {"factor": 2.0, "original": 100, "fast": 32.0, "slow": 1.0}),
               attn(2, 1, 8, 0.4, 4, moe(8, 3, 2, 2.0, 8), 1e5))
    tensors = make_tensors(cfg, 3)
    for name in ("l0.mix.q.norm", "l0.mix.k.norm"):
        tensors[name] = tensors[name] * 2.0               # scores that stand out
    model, _ = load(tmp_path, cfg, tensors)
    seq = [t % 60 for t in ids(300, 60, 8)]
    for at in (0, 1, 150):
        seq[at] = 63                                      # a rare token: a key of its own
    want = plain.forward(cfg, tensors, seq)
    assert err(logits(model, seq)[0], want) < 2 * TOL
    assert err(fed(model, seq, 290), want) < 2 * TOL
    for at in (0, 1, 150):
        other = list(seq)
        other[at] = 62
        moved = logits(model, other)[0]
        assert err(moved[max(at, 290):], want[max(at, 290):]) > 10 * TOL
        assert at == 0 or err(moved[:at], want[:at]) < 2 * TOL


def test_every_head_hears_every_other(tmp_path):
    """One entry of the mix at a time: it counts in prompts and in decoding."""
    cfg = case(64, 24, 1e-5, 2, 8, attn(4, 2, 8, 0.5, 4, None))
    tensors = make_tensors(cfg, 6)
    seq = ids(30, 64, 9)
    base = plain.forward(cfg, tensors, seq)
    for h in range(4):
        for g in range(4):
            changed = dict(tensors)
            talk = tensors["l0.mix.talk"].clone()
            talk[h, g] += 2.0
            changed["l0.mix.talk"] = talk
            want = plain.forward(cfg, changed, seq)
            assert err(want, base) > 20 * TOL
            model, _ = load(tmp_path, cfg, changed)
            assert err(logits(model, seq)[0], want) < TOL and err(fed(model, seq, 12), want) < TOL


# ---------------------------------------------------------------------------------------------------- framework paths
def plain_greedy(cfg, tensors, seq, n):
    seq = list(seq)
    for _ in range(n):
        seq.append(int(plain.forward(cfg, tensors, seq)[-1].argmax()))
    return seq


@pytest.mark.parametrize("name", ["mixed", "odd", "heads64"])
def test_greedy_generation_through_generate_and_the_graph_decoder(tmp_path, name):
    cfg = CASES[name]
    model, tensors = load(tmp_path, cfg)
    prompts = [ids(9, cfg["vocab"], 11), ids(9, cfg["vocab"], 12)]
    want = torch.tensor([plain_greedy(cfg, tensors, p, 8) for p in prompts])
    kw = dict(max_new_tokens=8, eos_token_id=None, pad_token_id=None)
    assert torch.equal(model.generate(torch.tensor(prompts), **kw), want)
    assert torch.equal(model.generate(torch.tensor(prompts), use_static_cache=False, **kw), want)
    dec = GraphedGreedyDecoder(model, max_len=40, use_graph=False)
    for _ in range(2):                                    # the decoder's cache and states are reused
        assert torch.equal(dec.generate(torch.tensor(prompts), 8), want)
    # unequal prompts, padded on the left
    short = prompts[1][:4]
    padded = torch.tensor([prompts[0], [0] * 5 + short])
    mask = torch.tensor([[1] * 9, [0] * 5 + [1] * 4])
    got = model.generate(padded, attention_mask=mask, **kw)
    assert got[0].tolist() == want[0].tolist() and got[1, 5:].tolist() == plain_greedy(cfg, tensors, short, 8)


def test_long_decoding_keeps_agreeing(tmp_path):
    cfg = CASES["mixed"]
    model, tensors = load(tmp_path, cfg)
    seq = ids(160, 96, 5)
    assert err(fed(model, seq, 2), plain.forward(cfg, tensors, seq)) < 2 * TOL


def test_sampling_and_beam_search(tmp_path):
    cfg = CASES["mixed"]
    model, _ = load(tmp_path, cfg)
    x = torch.tensor([ids(6, 96, 13)])
    torch.manual_seed(0)
    a = model.generate(x, do_sample=True, top_k=5, max_new_tokens=8, num_return_sequences=3, eos_token_id=None, pad_token_id=0)
    assert a.shape == (3, 14)
    got = model.generate(x, num_beams=3, max_new_tokens=8, eos_token_id=None, pad_token_id=0, return_dict_in_generate=True)
    lp = torch.log_softmax(logits(model, got.sequences[0].tolist())[0].double(), -1)
    score = sum(float(lp[t - 1, int(got.sequences[0, t])]) for t in range(6, 14)) / 14
    assert abs(score - float(got.sequences_scores[0])) < 1e-3
    again = model.generate(x, num_beams=3, max_new_tokens=8, eos_token_id=None, pad_token_id=0, use_cache=False)
    assert torch.equal(again, got.sequences)


def test_training_step_and_checkpointing(tmp_path):
    cfg = CASES["mixed"]
    model, _ = load(tmp_path, cfg)
    model.train()
    x = torch.tensor([ids(40, 96, 14), ids(40, 96, 15)])
    mask = torch.ones_like(x)
    mask[1, :11] = 0
    model(input_ids=x, labels=x, attention_mask=mask).loss.backward()
    grads = {n: p.grad.clone() for n, p in model.named_parameters()}
    assert all(torch.isfinite(g).all() and g.abs().sum() > 0 for g in grads.values())
    model.zero_grad()
    model.gradient_checkpointing_enable()
    model(input_ids=x, labels=x, attention_mask=mask).loss.backward()
    for n, p in model.named_parameters():
        assert torch.allclose(p.grad, grads[n], atol=1e-5), n


def test_registry_and_loading(tmp_path):
    cfg = CASES["mixed"]
    tensors = make_tensors(cfg)
    model, _ = load(tmp_path / "a", cfg, tensors)
    assert type(model) is ob.MasezenForCausalLM and model.config.vocab_size == 96 and model.config.num_hidden_layers == 4
    model.save_pretrained(str(tmp_path / "b"))
    again = ob.load_causal_lm(str(tmp_path / "b"))
    seq = ids(8, 96)
    assert torch.equal(logits(again, seq), logits(model, seq))
    fresh = ob.MasezenForCausalLM(ob.MasezenConfig(**cfg))
    assert fresh(input_ids=torch.tensor([seq])).logits.isfinite().all()
    cls = ob.MasezenForSequenceClassification.from_pretrained(str(tmp_path / "b"))
    assert cls(input_ids=torch.tensor([seq])).logits.shape == (1, 2)
    with pytest.raises(ValueError, match="input_ids"):
        model(inputs_embeds=torch.zeros(1, 3, 48))
    for change, exc in ((lambda t: t.pop("l0.mix.k"), KeyError), (lambda t: t.update({"l9.x": torch.zeros(1)}), KeyError),
                        (lambda t: t.update({"l1.mix.o": torch.zeros(48, 33)}), ValueError), (lambda t: t.pop("l1.mlp.e3.gate"), KeyError),
                        (lambda t: t.update({"l2.mix.talk": torch.zeros(2, 3)}), ValueError), (lambda t: t.pop("l2.canon1"), KeyError),
                        (lambda t: t.update({"l1.norm1": torch.zeros(48)}), ValueError), (lambda t: t.pop("side.embed"), KeyError),
                        (lambda t: t.update({"l2.ls2": torch.zeros(48)}), KeyError)):
        t = dict(tensors)
        change(t)
        write_model(str(tmp_path / "c"), cfg, t)
        with pytest.raises(exc):
            ob.load_causal_lm(str(tmp_path / "c"))
    with pytest.raises(NotImplementedError):
        model._exec_both_engines(tensor_parallel_size=2)


def test_configurations_that_nothing_implements_are_refused():
    ob.MasezenConfig(**CASES["mixed"])
    a = attn(2, 1, 8, 1.0, 4, None)
    without = lambda key: {**a, "mixer": {k: v for k, v in a["mixer"].items() if k != key}}     # noqa: E731
    wide = {**a, "mixer": {**a["mixer"], "vdim": 16}}
    for layer in ({"type": "window", "mixer": {}, "mlp": None}, attn(3, 2, 8, 1.0, 4, None), attn(2, 1, 8, 1.0, 10, None), attn(2, 1, 8, 1.0, 3, None),
                  wide, without("rot"), without("scale"), attn(2, 1, 8, 1.0, 4, {"kind": "gated", "ff": 3}), attn(2, 1, 8, 1.0, 4, moe(4, 2, 3, 1.0)),
                  attn(2, 1, 8, 1.0, 4, moe(4, 2, 0, 1.0)), attn(2, 1, 8, 1.0, 4, None, 10.0, {"factor": 2.0})):
        with pytest.raises(ValueError):
            ob.MasezenConfig(layers=[layer], norm={"eps": 1e-5}, vocab=8, width=8)
    for bad in ({"canon": {"taps": 0}}, {"token_side": {"dim": 0}}):
        with pytest.raises(ValueError):
            ob.MasezenConfig(layers=[a], vocab=8, width=8, **bad)


def test_trace_runner(tmp_path):
    """Two batches, one after the other; requests that end early; a step in which nothing is wanted."""
    import numpy as np
    cfg = CASES["odd"]
    model, _ = load(tmp_path / "m", cfg)
    a, b, c = ids(19, 51, 20), ids(4, 51, 21), ids(6, 51, 22)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": a[:17], "want": [0, 16]}, {"id": "b", "tokens": b[:3], "want": [1]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[3:], "want": [0]}, {"id": "a", "tokens": a[17:18], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[18:], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "c", "tokens": c[:5], "want": []}], "end": []},
             {"step": 4, "entries": [{"id": "c", "tokens": c[5:], "want": [0]}], "end": ["c"]}]
    out = tmp_path / "out"
    out.mkdir()
    run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(out),
                          "--max-tokens", "64", "--device", "cpu"], input="".join(json.dumps(x) + "\n" for x in lines), text=True,
                         capture_output=True)
    assert run.returncode == 0, run.stderr
    assert [x for x in run.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(5)]
    la, lb, lc = (logits(model, s)[0] for s in (a, b, c))
    want = {0: [la[0], la[16], lb[1]], 1: [lb[3], la[17]], 2: [la[18]], 4: [lc[5]]}
    assert sorted(os.listdir(out)) == [f"{i}.f32" for i in sorted(want)]
    for i, rows in want.items():
        got = torch.from_numpy(np.fromfile(str(out / f"{i}.f32"), dtype="<f4").reshape(len(rows), 51))
        assert err(got, torch.stack(rows)) < TOL, i


def test_generate_command_line(tmp_path):
    cfg = case(256, 24, 1e-5, 3, 8, attn(2, 1, 8, 0.4, 4, moe(16, 3, 2, 2.0, 8)), attn(2, 2, 8, 0.4, 8, dense(32), 1e4, YARN))
    model, _ = load(tmp_path, cfg)
    prompts = ["a b", "longer prompt"]
    run = subprocess.run(["python3", os.path.join(ROOT, "examples", "generate.py"), "--model", "auto", "--checkpoint", str(tmp_path),
                          "--prompt", *prompts, "--max-new-tokens", "6"], capture_output=True,
                         env={**os.environ, "CUDA_VISIBLE_DEVICES": "", "PYTHONPATH": ROOT})
    assert run.returncode == 0, run.stderr.decode()[-600:]
    want = b""
    for p in prompts:
        row = model.generate(torch.tensor([list(p.encode())]), max_new_tokens=6, eos_token_id=None, pad_token_id=None)[0]
        want += bytes(row.tolist()).decode("utf-8", "replace").encode() + b"\n"
    assert run.stdout == want
