"""Begovik on the CPU statements of the ops: every mechanism against ``plain_begovik.py`` (double precision, loops), the cache and
the states under decoding, portions, padded batches, reordering and reuse, the scheduler and sampling paths of
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
from oslo_b200.models.mixers import (BonusRecurrence, DecayedLinearAttention, GatedMLP, GroupedQueryAttention, SelectiveScan,
                                     SideBySide)

from . import plain_begovik as plain
from .begovik_cases import CASES, attn, case, dense, far_key_weights, lin, make_tensors, mamba, parallel, public, wkv, write_model

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = 3e-5


def load(tmp_path, cfg, tensors=None, seed=0, dtype=torch.float32):
    tensors = make_tensors(cfg, seed) if tensors is None else tensors
    write_model(str(tmp_path), cfg, tensors)
    return ob.load_causal_lm(str(tmp_path), torch_dtype=dtype).eval(), tensors


def ids(n, vocab, seed=1):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def err(a, b):
    b = b.double()
    return float((a.double() - b).abs().max() / b.abs().max().clamp(min=1e-6))


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
def test_head_norm_comes_before_the_interleaved_rotation_of_the_first_dims():
    n, heads, dim, eps = 7, 3, 10, 1e-2
    x, w = torch.randn(1, n, heads, dim), torch.randn(dim)
    pos = torch.arange(n)[None]
    for rot in (0, 4, 10):
        freq = torch.tensor(ops.reference.rotary_frequencies(rot, 50.0))
        got = ops.reference.norm_rotate(x, w, eps, pos, freq)
        assert err(got[0], plain.rotate(plain.norm(x[0].double(), w.double(), eps), rot, 50.0)) < TOL
        assert err(got[..., rot:][0] if rot < dim else torch.ones(1), plain.norm(x[0].double(), w.double(), eps)[..., rot:]
                   if rot < dim else torch.ones(1)) < TOL
    # a rotated query and key see their distance only
    q, k = (plain.rotate(torch.randn(1, 1, 6, dtype=torch.float64).expand(40, 1, 6), 6, 30.0)[:, 0] for _ in range(2))
    assert abs(float(q[9] @ k[4]) - float(q[39] @ k[34])) < 1e-9


@pytest.mark.parametrize("heads,groups", [(1, 1), (4, 2), (6, 1), (3, 3)])
def test_grouped_attention_with_cap_and_zero_sink(heads, groups):
    n, dim, vdim, scale, cap = 9, 8, 5, 0.7, 2.5
    q, k, v = torch.randn(1, n, heads, dim), torch.randn(1, n, groups, dim), torch.randn(1, n, groups, vdim)
    k[0, 2] *= 8.0                                        # beyond the cap
    zero = torch.zeros(heads)
    want = plain.capped_attention(q[0].double(), k[0].double(), v[0].double(), scale, cap)
    got, probs = ops.reference.sink_attention(q, k, v, None, zero, None, scale, cap)
    assert err(got.view(n, heads, vdim), want) < TOL
    # the first token's weight is e / (1 + e), never 1
    s = cap * math.tanh(float(q[0, 0, -1] @ k[0, 0, -1]) * scale / cap)
    assert abs(float(probs[0, -1, 0, 0]) - math.exp(s) / (1.0 + math.exp(s))) < 1e-5
    # the last queries of a longer sequence, and one query over a cache with room
    tail, _ = ops.reference.sink_attention(q[:, 6:], k, v, None, zero, None, scale, cap)
    assert err(tail, got[6:]) < 1e-6
    kc, vc = torch.full((1, groups, n + 4, dim), float("nan")), torch.full((1, groups, n + 4, vdim), float("nan"))
    kc[:, :, :n], vc[:, :, :n] = k.transpose(1, 2), v.transpose(1, 2)
    kc[:, :, n:] = 1e4
    one = ops.reference.grouped_decode(q[:, -1], kc, vc, torch.tensor([n]), None, zero, scale, cap)
    assert err(one, got[-1:]) < 1e-5
    # a padded key is out of the softmax
    keep = torch.ones(1, n, dtype=torch.uint8)
    keep[0, :3] = 0
    got, _ = ops.reference.sink_attention(q, k, v, keep, zero, None, scale, cap)
    want = plain.capped_attention(q[0, 3:].double(), k[0, 3:].double(), v[0, 3:].double(), scale, cap)
    assert err(got.view(n, heads, vdim)[3:], want) < TOL


@pytest.mark.parametrize("heads,dim,vdim", [(1, 4, 6), (3, 10, 5), (2, 16, 16)])
def test_recurrences_are_the_token_by_token_rules(heads, dim, vdim):
    n = 11
    q, k, v = torch.randn(n, heads * dim), torch.randn(n, heads * dim), torch.randn(n, heads * vdim)
    decay = torch.tensor([0.9, 0.0, 1.0][:heads])
    keep = torch.tensor([[0, 0, 0, 1, 1, 1, 1, 1, 1, 1, 1]])
    sel = keep[0].bool()
    shaped = lambda t, rows: t.double()[rows].view(-1, heads, t.size(1) // heads)               # noqa: E731
    s0 = torch.randn(1, heads, dim, vdim)
    for kp, rows in ((None, torch.ones(n, dtype=torch.bool)), (keep, sel)):
        want, end = plain.decayed_sum(*(plain.silu(shaped(t, rows)) for t in (q, k, v)), decay.double(), s0[0].double())
        got, state = ops.reference.decayed_attention(q, k, v, decay, kp, s0, 1, heads)
        assert err(got[0][rows], want) < TOL and err(state[0], end) < TOL and not got[0][~rows].any()
    z, w0, u = torch.randn(n, heads * dim), torch.randn(heads * dim) - 1.0, torch.randn(heads * dim)
    w = torch.exp(-torch.exp(z.double() + w0.double()))
    s0 = torch.randn(1, heads, dim, dim)
    v = torch.randn(n, heads * dim)
    for kp, rows in ((None, torch.ones(n, dtype=torch.bool)), (keep, sel)):
        want, end = plain.bonus_recurrence(*(shaped(t, rows) for t in (q, k, v)), shaped(w, rows), u.double().view(heads, dim), s0[0].double())
        got, state = ops.reference.bonus_recurrence(q, k, v, z, w0, u, kp, s0, 1, heads)
        assert err(got[0][rows], want) < TOL and err(state[0], end) < TOL and not got[0][~rows].any()


def test_bonus_counts_for_the_current_token_only():
    heads, dim = 1, 4
    r, k, v, z = torch.ones(2, dim), torch.eye(2, dim), torch.tensor([[1.0, 0, 0, 0], [0, 1.0, 0, 0]]), torch.zeros(2, dim)
    w0, u = torch.full((dim,), -50.0), torch.full((dim,), 7.0)          # no decay, a large bonus
    o, s = ops.reference.bonus_recurrence(r, k, v, z, w0, u, None, None, 1, heads)
    assert torch.allclose(o[0, 0, 0], torch.tensor([7.0, 0, 0, 0])) and torch.allclose(o[0, 1, 0], torch.tensor([1.0, 7.0, 0, 0]))
    assert torch.allclose(s[0, 0, 0], torch.tensor([1.0, 0, 0, 0])) and torch.allclose(s[0, 0, 1], torch.tensor([0, 1.0, 0, 0]))


def test_token_shift_and_convolution_look_back_to_the_state():
    batch, n, width, taps = 2, 6, 5, 4
    h, mu = torch.randn(batch * n, width), torch.rand(3, width)
    prev = torch.randn(batch, width)
    got, last = ops.reference.token_shift(h, mu, batch, None, prev)
    hb = h.double().view(batch, n, width)
    for b in range(batch):
        before = plain.shifted(hb[b], prev[b].double())
        for i in range(3):
            assert err(got.view(3, batch, n, width)[i, b], hb[b] + (before - hb[b]) * mu[i].double()) < TOL
    assert torch.equal(last, h.view(batch, n, width)[:, -1])
    w, bias, back = torch.randn(width, taps), torch.randn(width), torch.randn(batch, taps - 1, width)
    for m in (n, 2, 1):                                   # also fewer tokens than the convolution is wide
        x = torch.randn(batch * m, width)
        got, last = ops.reference.causal_conv(x, w, bias, batch, None, back, silu=True)
        for b in range(batch):
            want = plain.silu(plain.causal_conv(x.double().view(batch, m, width)[b], w.double(), bias.double(), back[b].double()))
            assert err(got.view(batch, m, width)[b], want) < TOL
            assert torch.equal(last[b], torch.cat([back[b], x.view(batch, m, width)[b]])[-(taps - 1):])
    keep = torch.tensor([[0, 0, 1, 1, 1, 1], [1, 1, 1, 1, 1, 1]])         # the first real token has zeros before it
    got, _ = ops.reference.token_shift(h, mu, batch, keep, None)
    alone, _ = ops.reference.token_shift(h[2:n], mu, 1, None, None)
    assert err(got.view(3, batch, n, width)[:, 0, 2:], alone.view(3, n - 2, width)) < 1e-6


def test_selective_scan_is_the_token_by_token_rule():
    n, c, s = 10, 6, 4
    x, dt, z = torch.randn(n, c), torch.randn(n, c), torch.randn(n, c)
    bias, a_log, b, cc, d = torch.randn(c), torch.randn(c, s), torch.randn(n, s), torch.randn(n, s), torch.randn(c)
    s0 = torch.randn(1, c, s)
    want, end = plain.selective_scan(x.double(), plain.softplus(dt.double() + bias.double()), -torch.exp(a_log.double()), b.double(),
                                     cc.double(), d.double(), s0[0].double())
    got, state = ops.reference.selective_scan(x, dt, bias, a_log, b, cc, d, z, 1, None, s0)
    assert err(got, want * plain.silu(z.double())) < TOL and err(state[0], end) < TOL
    keep = torch.tensor([[0] * 4 + [1] * 6])
    want, end = plain.selective_scan(x[4:].double(), plain.softplus(dt[4:].double() + bias.double()), -torch.exp(a_log.double()),
                                     b[4:].double(), cc[4:].double(), d.double())
    got, state = ops.reference.selective_scan(x, dt, bias, a_log, b, cc, d, z, 1, keep, None)
    assert err(got[4:], want * plain.silu(z[4:].double())) < TOL and err(state[0], end) < TOL
    # steps of any size: softplus neither overflows nor loses small values
    big = torch.tensor([[-90.0, -20.0, 0.0, 15.0, 40.0, 200.0]]).expand(2, 6).contiguous()
    out, state = ops.reference.selective_scan(torch.ones(2, 6), big, torch.zeros(6), torch.zeros(6, 1), torch.ones(2, 1), torch.ones(2, 1),
                                              torch.zeros(6), torch.ones(2, 6), 1, None, None)
    want, _ = plain.selective_scan(torch.ones(2, 6).double(), plain.softplus(big.double()), -torch.ones(6, 1).double(), torch.ones(2, 1).double(),
                                   torch.ones(2, 1).double(), torch.zeros(6).double())
    assert torch.isfinite(out).all() and torch.allclose(out.double(), want * plain.silu(torch.ones(2, 6).double()), rtol=1e-5, atol=1e-30)


def test_clamped_unit():
    limit = 0.8
    g, u = torch.tensor([-9.0, -0.5, 0.3, 0.79, 0.81, 5.0]), torch.tensor([-3.0, -0.81, -0.2, 0.5, 0.9, 7.0])
    assert err(ops.clamped_glu(g[None], u[None], limit, 1.702)[0], plain.clamped_glu(g.double(), u.double(), limit)) < TOL
    assert float(ops.clamped_glu(torch.tensor([[-9.0]]), torch.tensor([[0.0]]), limit, 1.702)) != 0.0      # only cut from above
    m = randomise(GatedMLP(12, 20, limit=limit))
    get = getter({"gate": m.in_proj.part("gate"), "up": m.in_proj.part("up"), "down": m.down.weight})
    h = torch.randn(9, 12)
    assert err(m(h).y.detach(), plain.dense_mlp(h.double(), get, limit)) < TOL


def test_branch_join_norms_scales_and_adds():
    x, y, ws = torch.randn(6, 10), torch.randn(3, 6, 10), torch.randn(4, 10)
    d = lambda t: t.double()                                                                    # noqa: E731
    want = d(x) + 0.3 * (0.5 * (plain.norm(d(y[0]), d(ws[0]), 1e-3) + plain.norm(d(y[1]), d(ws[1]), 1e-3)) + d(y[2]))
    got, (h1, h2) = ops.branch_join(x, [(y[0], ws[0], 0.5), (y[1], ws[1], 0.5), (y[2], None, 1.0)], 0.3, 1e-3, [ws[2], ws[3]])
    assert err(got, want) < TOL and err(h1, plain.norm(want, d(ws[2]), 1e-3)) < TOL and err(h2, plain.norm(want, d(ws[3]), 1e-3)) < TOL


def test_mixers_alone():
    width, n, eps = 18, 9, 1e-3
    h = torch.randn(n, width)
    pos = torch.arange(n)[None]
    with torch.no_grad():
        a = randomise(GroupedQueryAttention(width, 4, 2, 8, 6, 0.4, eps, rot_dims=4, rot_base=100.0, softcap=3.0))
        get = getter({**{s: a.in_proj.part(s) for s in "qkv"}, "q.norm": a.q_norm.weight, "k.norm": a.k_norm.weight, "o": a.out_proj.weight})
        m = attn(4, 2, 8, 6, 0.4, 3.0, 4, 100.0)
        assert err(a(h, 1, 0, None, None, pos).y, plain.attention(h.double(), get, m, eps)) < TOL
        b = randomise(DecayedLinearAttention(width, 3, 5, 4, [0.2, 0.9, 1.0], eps))
        get = getter({**{s: b.in_proj.part(s) for s in "qkvg"}, "norm": b.o_norm.weight, "o": b.out_proj.weight})
        assert err(b(h, 1, 0, None, None).y, plain.lightning(h.double(), get, lin(3, 5, 4, (0.2, 0.9, 1.0)), eps)[0]) < TOL
        c = randomise(BonusRecurrence(width, 3, 6, eps, decay_rank=4))
        get = getter({**{f"mu.{s}": c.mu[i] for i, s in enumerate("rkvgw")}, **{s: c.rkvg.weight[i] for i, s in enumerate("rkvg")},
                      "w1": c.w1.weight, "w2": c.w2.weight, "w0": c.w0, "u": c.u, "norm": c.o_norm, "o": c.out_proj.weight})
        assert err(c(h, 1, 0, None, None).y, plain.wkv(h.double(), get, {"heads": 3, "dim": 6}, eps)[0]) < TOL
        s = randomise(SelectiveScan(width, 10, 4, 3, 3))
        packed = lambda p, names: torch.cat([p.part(i) for i in names])                         # noqa: E731
        get = getter({"in": packed(s.in_proj, ("x", "z")), "conv": s.conv_weight, "conv.b": s.conv_bias, "x": packed(s.x_proj, ("dt", "b", "c")),
                      "dt": s.dt_proj.weight, "dt.b": s.dt_bias, "A_log": s.a_log, "D": s.d, "o": s.out_proj.weight})
        m = {"inner": 10, "state": 4, "dt_rank": 3, "conv": 3}
        assert err(s(h, 1, 0, None, None).y, plain.mamba1(h.double(), get, m, eps)[0]) < TOL
        two = SideBySide(width, dict(heads=4, kv_heads=2, dim=8, vdim=6, scale=0.4), dict(heads=3, dim=5, vdim=4, decay=[0.5] * 3), eps)
        out = two(h, 1, 0, None, None, pos)
        assert out.y is None and [b.factor for b in out.branches] == [0.5, 0.5] and all(b.weight is not None for b in out.branches)


# ---------------------------------------------------------------------------------------------------- the whole model
@pytest.mark.parametrize("name", sorted(CASES))
def test_logits_and_residual_stream(tmp_path, name):
    cfg = CASES[name]
    if name == "ones":                                    # without cap: compare with a cap that does nothing
        cfg = json.loads(json.dumps(cfg))
        cfg["layers"][0]["mixer"]["left"].update(softcap=1e9, rot={"dims": 0, "base": 1.0})
    model, tensors = load(tmp_path, CASES[name])
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
    assert err(out.logits[0], want) < TOL and out.past_key_values is None
    assert [p is not None for p in out.attentions] == [l["type"] == "parallel" for l in cfg["layers"]]


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
    d = out.logits[0].double() - want
    assert float(d.pow(2).mean().sqrt() / want.pow(2).mean().sqrt()) < 0.08


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
    # only what the design says is kept: keys and values of attention layers, one state per recurrence, what a shift or a
    # convolution looks back to
    kinds = [l["type"] for l in cfg["layers"]]
    assert sorted(cache.k) == [i for i, k in enumerate(kinds) if k == "parallel"] and not cache.latent
    assert {k if isinstance(k, int) else k[0] for k in cache.state} == set(range(len(kinds)))
    assert {k for k in cache.state if not isinstance(k, int)} == {(i, {"wkv": "shift", "mamba1": "conv"}[k]) for i, k in enumerate(kinds)
                                                                   if k != "parallel"}


@pytest.mark.parametrize("name", ["mixed", "odd", "heads64"])
def test_batches_of_unequal_requests_match_each_alone(tmp_path, name):
    cfg = CASES[name]
    model, _ = load(tmp_path, cfg)
    seqs = [ids(n, cfg["vocab"], seed=n) for n in (24, 1, 13, 7)]
    alone = [logits(model, s)[0] for s in seqs]
    prompt = [18, 1, 9, 2]                                # the rest is fed token by token; shorter requests end earlier
    seqs[1] = seqs[1] + ids(3, cfg["vocab"], seed=99)
    alone[1] = logits(model, seqs[1])[0]
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


def test_keys_far_away_decide_the_output(tmp_path):
    """With attention sharpened to a search, a prompt's and a decoded token's result hang on single keys hundreds of tokens
    back: changing such a key's token changes the logits, and all ways of feeding the sequence agree with the plain model."""
    cfg = case(64, 40, 1e-5, parallel(attn(2, 1, 16, 24, 1.0, 30.0, 4, 1e5), lin(1, 4, 8, (0.5,)), None), mamba(16, 4, 4, 2, dense(24)))
    tensors = far_key_weights(0, make_tensors(cfg, 3), 2.0)
    model, _ = load(tmp_path, cfg, tensors)
    seq = [t % 60 for t in ids(300, 60, 8)]
    for at in (0, 1, 150):
        seq[at] = 63                                      # a rare token: a key of its own
    want = plain.forward(cfg, tensors, seq)
    assert err(logits(model, seq)[0], want) < 2 * TOL
    cache = StaticKVCache(320)
    with torch.no_grad():
        model(input_ids=torch.tensor([seq[:290]]), past_key_values=cache)
        got = torch.cat([model(input_ids=torch.tensor([[t]]), past_key_values=cache).logits[0] for t in seq[290:]])
    assert err(got, want[290:]) < 2 * TOL
    for at in (0, 1, 150):
        other = list(seq)
        other[at] = 62
        moved = logits(model, other)[0]
        assert err(moved[max(at, 290):], want[max(at, 290):]) > 20 * TOL
        assert at == 0 or err(moved[:at], want[:at]) < 2 * TOL


@pytest.mark.parametrize("kind", ["wkv", "mamba1", "lightning"])
def test_states_carry_the_first_tokens_through_a_long_prompt(tmp_path, kind):
    if kind == "wkv":
        cfg = case(64, 24, 1e-5, wkv(2, 12, None), wkv(1, 8, dense(16)))
        tensors = make_tensors(cfg, 4)
        for i in range(2):
            tensors[f"l{i}.mix.w0"] = tensors[f"l{i}.mix.w0"] - 6.0         # hardly forgets
    elif kind == "mamba1":
        cfg = case(64, 24, 1e-5, mamba(32, 8, 4, 4, None), mamba(16, 4, 4, 3, dense(16)))
        tensors = make_tensors(cfg, 4)
        for i in range(2):
            tensors[f"l{i}.mix.A_log"] = tensors[f"l{i}.mix.A_log"] - 6.0
    else:
        cfg = case(64, 24, 1e-5, parallel(attn(2, 1, 8, 8, 0.01, 1.0, 4), lin(2, 8, 8, (0.999, 1.0)), None))
        tensors = make_tensors(cfg, 4)
    model, _ = load(tmp_path, cfg, tensors)
    seq = ids(260, 64, 9)
    want = plain.forward(cfg, tensors, seq)
    assert err(logits(model, seq)[0], want) < TOL
    other = [(seq[0] + 1) % 64] + seq[1:]
    assert err(logits(model, other)[0, -1], want[-1]) > 3 * TOL


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
    x = torch.tensor([ids(12, 96, 14)])
    model(input_ids=x, labels=x).loss.backward()
    grads = {n: p.grad.clone() for n, p in model.named_parameters()}
    assert all(torch.isfinite(g).all() for g in grads.values()) and all(g.abs().sum() > 0 for g in grads.values())
    model.zero_grad()
    model.gradient_checkpointing_enable()
    model(input_ids=x, labels=x).loss.backward()
    for n, p in model.named_parameters():
        assert torch.allclose(p.grad, grads[n], atol=1e-6), n


def test_registry_and_loading(tmp_path):
    cfg = CASES["mixed"]
    tensors = make_tensors(cfg)
    model, _ = load(tmp_path / "a", cfg, tensors)
    assert type(model) is ob.BegovikForCausalLM and model.config.vocab_size == 96 and model.config.num_hidden_layers == 6
    model.save_pretrained(str(tmp_path / "b"))            # the ranks that only the weights fix are saved with it
    again = ob.load_causal_lm(str(tmp_path / "b"))
    seq = ids(8, 96)
    assert torch.equal(logits(again, seq), logits(model, seq))
    fresh = ob.BegovikForCausalLM(ob.BegovikConfig(**public(cfg)))
    assert fresh(input_ids=torch.tensor([seq])).logits.isfinite().all()
    cls = ob.BegovikForSequenceClassification.from_pretrained(str(tmp_path / "b"))
    assert cls(input_ids=torch.tensor([seq])).logits.shape == (1, 2)
    for change, exc in ((lambda t: t.pop("l0.mix.left.k"), KeyError), (lambda t: t.update({"l9.x": torch.zeros(1)}), KeyError),
                        (lambda t: t.update({"l1.mix.o": torch.zeros(48, 33)}), ValueError),
                        (lambda t: t.update({"l2.mix.x": torch.zeros(41, 64)}), ValueError), (lambda t: t.pop("l1.mix.mu.g"), KeyError)):
        t = dict(tensors)
        change(t)
        write_model(str(tmp_path / "c"), cfg, t)
        with pytest.raises(exc):
            ob.load_causal_lm(str(tmp_path / "c"))
    with pytest.raises(NotImplementedError):
        model._exec_both_engines(tensor_parallel_size=2)


def test_configurations_that_nothing_implements_are_refused():
    good = public(CASES["mixed"])
    ob.BegovikConfig(**good)
    a, b = attn(2, 1, 8, 8, 1.0, 1.0, 4), lin(2, 8, 8, (0.5, 0.5))
    for layer in ({"type": "window", "mixer": {}, "mlp": None}, parallel(attn(3, 2, 8, 8, 1.0, 1.0, 4), b, None),
                  parallel(a, lin(2, 8, 8, (0.5,)), None), parallel(attn(2, 1, 8, 8, 1.0, 1.0, 10), b, None), parallel(attn(2, 1, 8, 8, 1.0, 1.0, 3), b, None),
                  parallel(a, {"heads": 1}, None), {"type": "wkv", "mixer": {"heads": 1}, "mlp": None},
                  mamba(8, 2, 2, 2, {"kind": "moe"}), mamba(8, 2, 2, 2, {"kind": "dense", "ff": 3})):
        with pytest.raises(ValueError):
            ob.BegovikConfig(layers=[layer], norm={"eps": 1e-5}, vocab=8, width=8)


def test_trace_runner(tmp_path):
    """Two batches, one after the other; requests that end early; a step in which nothing is wanted."""
    import numpy as np
    cfg = CASES["odd"]
    model, _ = load(tmp_path / "m", cfg)
    a, b, c = ids(9, 51, 20), ids(4, 51, 21), ids(6, 51, 22)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": a[:7], "want": [0, 6]}, {"id": "b", "tokens": b[:3], "want": [1]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[3:], "want": [0]}, {"id": "a", "tokens": a[7:8], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[8:], "want": [0]}], "end": ["a"]},
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
    want = {0: [la[0], la[6], lb[1]], 1: [lb[3], la[7]], 2: [la[8]], 4: [lc[5]]}
    assert sorted(os.listdir(out)) == [f"{i}.f32" for i in sorted(want)]
    for i, rows in want.items():
        got = torch.from_numpy(np.fromfile(str(out / f"{i}.f32"), dtype="<f4").reshape(len(rows), 51))
        assert err(got, torch.stack(rows)) < TOL, i


def test_generate_command_line(tmp_path):
    cfg = case(256, 24, 1e-5, wkv(2, 8, dense(16)), parallel(attn(2, 1, 8, 8, 0.4, 5.0, 4), lin(2, 8, 8, (0.5, 0.9)), dense(32)),
               mamba(32, 4, 4, 4, None))
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
