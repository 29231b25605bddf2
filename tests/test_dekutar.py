"""Dekutar on the CPU statements of the ops: every mechanism against ``plain_dekutar.py`` (double precision, loops), the cache and
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
from oslo_b200.models.mixers import GroupedQueryAttention, HyperConnections, LatentAttention, MatrixMemory, MixtureOfExperts
from oslo_b200.ops.reference import SublayerResult
from oslo_b200.parallel.layers import RMSNorm

from . import plain_dekutar as plain
from .dekutar_cases import CASES, attn, case, latent, make_tensors, mlstm, moe, write_model

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = 5e-5


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
def test_rotations_pair_what_they_say_and_see_distances_only():
    n, heads = 9, 2
    x = torch.randn(1, n, heads, 10)
    pos = torch.arange(n)[None]
    for dims in (2, 6, 10):
        freq = torch.tensor(ops.reference.rotary_frequencies(dims, 40.0))
        want = plain.rms(plain.rotate_interleaved(x[0].double(), dims, 40.0), 1e-2)
        assert err(ops.reference.norm_rotate(x, None, 1e-2, pos, freq)[0], want) < TOL     # the norm before or after is the same
        part = x[..., :dims]
        assert err(ops.reference.rotate_halves(part, pos, freq)[0], plain.rotate_halves(part[0].double(), dims, 40.0)) < TOL
    q, k = (torch.randn(1, 1, 6, dtype=torch.float64).expand(40, 1, 6) for _ in range(2))
    for turn in (plain.rotate_interleaved, plain.rotate_halves):
        a, b = turn(q, 6, 30.0)[:, 0], turn(k, 6, 30.0)[:, 0]
        assert abs(float(a[9] @ b[4]) - float(a[39] @ b[34])) < 1e-9
    assert err(plain.rotate_halves(q[5:], 6, 30.0, first=5), plain.rotate_halves(q, 6, 30.0)[5:]) < 1e-12


@pytest.mark.parametrize("size,keep_first", [(1, 0), (1, 3), (4, 0), (4, 2), (7, 30), (5, 4), (30, 2), (11, 1)])
@pytest.mark.parametrize("heads,groups", [(1, 1), (6, 2)])
def test_windows_and_kept_keys(size, keep_first, heads, groups):
    n, dim, vdim, scale = 23, 6, 5, 0.4
    q, k, v = torch.randn(1, n, heads, dim), torch.randn(1, n, groups, dim), torch.randn(1, n, groups, vdim)
    want = plain.softmax_attention(q[0].double(), k[0].double(), v[0].double(), scale, size, keep_first).reshape(n, -1)
    args = dict(window=size, keep_first=keep_first)
    got, probs = ops.reference.sink_attention(q, k, v, None, None, None, scale, **args)
    assert err(got, want) < TOL
    for i in range(n):
        assert [bool(p > 0) for p in probs[0, 0, i]] == [plain.sees(i, j, size, keep_first) for j in range(n)]
    tail, _ = ops.reference.sink_attention(q[:, 15:], k, v, None, None, None, scale, **args)
    assert err(tail, got[15:]) < 1e-6
    kc, vc = torch.full((1, groups, n + 4, dim), 1e4), torch.full((1, groups, n + 4, vdim), float("nan"))
    for last in (0, size - 1, size, min(n - 1, size + keep_first), n - 1):
        if last >= n:
            continue
        kc[:, :, :last + 1], vc[:, :, :last + 1] = k[:, :last + 1].transpose(1, 2), v[:, :last + 1].transpose(1, 2)
        kc[:, :, last + 1:], vc[:, :, last + 1:] = 1e4, float("nan")
        one = ops.reference.grouped_decode(q[:, last], kc, vc, torch.tensor([last + 1]), None, None, scale, **args)
        assert err(one, got[last:last + 1]) < 1e-5
    # padding ahead of the sequence moves the kept keys along
    pad = 6
    front = lambda t: torch.cat([torch.randn(1, pad, *t.shape[2:]), t], dim=1)                  # noqa: E731
    keep, lead = torch.tensor([[0] * pad + [1] * n]), torch.tensor([pad], dtype=torch.int32)
    moved, _ = ops.reference.sink_attention(front(q), front(k), front(v), keep, None, None, scale, **args, lead=lead)
    assert err(moved[pad:], got) < 1e-5 and torch.isfinite(moved).all()
    one = ops.reference.grouped_decode(q[:, -1], front(k).transpose(1, 2), front(v).transpose(1, 2), torch.tensor([pad + n]), keep, None, scale,
                                       **args, lead=lead)
    assert err(one, got[-1:]) < 1e-5


def test_output_gates_per_head_and_per_element():
    n, heads, dim, vdim = 5, 3, 4, 2
    q, k, v = torch.randn(1, n, heads, dim), torch.randn(1, n, heads, dim), torch.randn(1, n, heads, vdim)
    o, _ = ops.reference.sink_attention(q, k, v, None, None, None, 1.0)
    for gate in (torch.randn(n, heads), torch.randn(n, heads * vdim)):
        g = torch.sigmoid(gate)
        g = g.repeat_interleave(vdim, dim=1) if gate.size(1) == heads else g
        got, _ = ops.reference.sink_attention(q, k, v, None, None, gate, 1.0)
        assert err(got, o * g) < 1e-6


def test_latent_decode_is_attention_over_expanded_keys():
    n, heads, dim, rot, vdim, rank, scale = 8, 3, 4, 6, 5, 7, 0.3
    c, shared = torch.randn(1, n, rank), torch.randn(1, n, rot)
    uk, uv = torch.randn(heads * dim, rank), torch.randn(heads * vdim, rank)
    pos, freq = torch.tensor([[n - 1]]), torch.tensor(ops.reference.rotary_frequencies(rot, 20.0))
    q, gate = torch.randn(1, heads * (dim + rot)), torch.randn(1, heads * vdim)
    turned = ops.reference.rotate_halves(q.view(1, 1, heads, -1)[..., dim:], pos, freq)
    want, _ = ops.reference.sink_attention(q.view(1, 1, heads, -1)[..., :dim], (c[0] @ uk.T).view(1, n, heads, dim), (c[0] @ uv.T).view(1, n, heads, vdim),
                                           None, None, gate, scale, q_rot=turned, k_rot=shared)
    room = torch.cat([torch.cat([c, shared], -1), torch.full((1, 3, rank + rot), 50.0)], dim=1)
    got = ops.latent_decode(q, uk, uv, room, torch.tensor([n]), None, None, gate, scale, heads, pos, freq)
    assert err(got, want) < TOL


@pytest.mark.parametrize("heads,dim,vdim,cap", [(1, 4, 6, 3.0), (3, 5, 2, 20.0), (2, 8, 8, 1.0)])
def test_matrix_memory_is_the_token_by_token_rule(heads, dim, vdim, cap):
    n = 13
    q, k, v = torch.randn(n, heads * dim), torch.randn(n, heads * dim), torch.randn(n, heads * vdim)
    z, bias = 8.0 * torch.randn(n, 2 * heads), torch.randn(2 * heads)
    gates = plain.capped(z.double() + bias.double(), cap)
    shaped = lambda t, rows: t.double()[rows].view(-1, heads, t.size(1) // heads)               # noqa: E731
    width = ops.reference.memory_state_width(vdim)
    s0, n0, m0 = torch.randn(heads, dim, vdim), torch.randn(heads, dim), torch.randn(heads)
    state = torch.zeros(1, heads, dim, width)
    state[0, :, :, :vdim], state[0, :, :, vdim] = s0, n0
    padded = torch.tensor([[0, 0, 0, 1, 1, 1, 1, 0, 1, 1, 1, 1, 1]])
    for keep in (None, padded):
        rows = torch.ones(n, dtype=torch.bool) if keep is None else keep[0].bool()
        for start in (None, (s0.double(), n0.double(), m0.double())):
            want, end = plain.matrix_memory(shaped(q, rows) * dim ** -0.5, shaped(k, rows), shaped(v, rows), gates[rows, :heads],
                                            plain.log_sigmoid(gates[rows, heads:]), start)
            o, nq, m, last, top = ops.reference.matrix_memory(q, k, v, z, bias, cap, keep, None if start is None else state,
                                                              None if start is None else m0[None], 1, heads)
            got = o.view(n, heads, vdim) / (torch.maximum(nq.abs(), torch.exp(-m)) + 1e-6)[..., None]
            assert err(got[rows], want) < TOL and not o[~rows].any()
            assert err(last[0, :, :, :vdim], end[0]) < TOL and err(last[0, :, :, vdim], end[1]) < TOL and err(top[0], end[2]) < TOL


def test_running_maximum_starts_at_zero():
    """A first token with a small input gate writes exp(i - 0), not 1."""
    one = torch.ones(1, 1)
    z, bias = torch.tensor([[-3.0, 50.0]]), torch.zeros(2)
    o, nq, m, state, top = ops.reference.matrix_memory(one, one, one, z, bias, 1e6, None, None, None, 1, 1)
    assert abs(float(m)) < 1e-6 and abs(float(o) - math.exp(-3.0)) < 1e-6 and abs(float(nq) - math.exp(-3.0)) < 1e-6
    want, _ = plain.matrix_memory(*(torch.ones(1, 1, 1, dtype=torch.float64),) * 3, torch.tensor([[-3.0]]).double(), torch.zeros(1, 1).double())
    assert abs(float(want) - math.exp(-3.0) / (1.0 + 1e-6)) < 1e-12


def test_normaliser_enters_before_the_head_norm():
    rows, heads, vdim = 4, 2, 3
    o, gate, w = torch.randn(rows, heads * vdim), torch.randn(rows, heads * vdim), torch.randn(heads * vdim)
    z, m = torch.randn(rows, heads), torch.randn(rows, heads)
    den = torch.maximum(z.abs(), torch.exp(-m)) + 1e-6
    want = plain.rms(o.double().view(rows, heads, vdim) / den.double()[..., None], 0.1).reshape(rows, -1) * w.double() * plain.sigmoid(gate.double())
    assert err(ops.gated_rms_norm(o, w, gate, 0.1, vdim, "sigmoid", (z, m)), want) < TOL


def test_routing_scores_choices_and_identity_outputs():
    n, width, experts, identity, top = 40, 6, 5, 3, 3
    h, w, corr = torch.randn(n, width), torch.randn(experts + identity, width), torch.randn(experts + identity)
    idx, weights = ops.moe_route(h, w, corr, top, scored=True)
    want_idx, want = plain.route(h.double(), w.double(), corr.double(), top)
    assert torch.equal(idx.long(), want_idx) and err(weights, want) < TOL and err(weights.sum(-1), torch.ones(n)) < 1e-5
    # the correction decides who is chosen, not with what weight
    high = torch.zeros(experts + identity)
    high[2] = 50.0
    idx, weights = ops.moe_route(h, w, high, 1, scored=True)
    assert bool((idx == 2).all()) and err(weights, torch.ones(n, 1)) < 1e-6
    module = randomise(MixtureOfExperts(width, 4, experts, top, unit="silu", scored=True, identity=identity, shared=7))
    with torch.no_grad():
        f = module(h)
        got = ops.reference.collect_result(SublayerResult(f.y, f.slots, f.weights, f.choice, experts, h, f.shared, f.shared_gate))
    s = module.shared
    table = {"router": module.router.weight, "correction": module.correction, "shared.sg": s.in_proj.part("sg"),
             "shared.gate": s.in_proj.part("gate"), "shared.up": s.in_proj.part("up"), "shared.down": s.down.weight}
    for e in range(experts):
        table.update({f"e{e}.gate": module.up[e, 0::2], f"e{e}.up": module.up[e, 1::2], f"e{e}.down": module.down[e]})
    mlp = {"router": {"experts": experts, "identity": identity, "top": top}}
    assert err(got, plain.moe(h.double(), getter(table), mlp)) < TOL
    assert bool((f.choice >= experts).any()) and bool((f.choice < experts).any())


@pytest.mark.parametrize("streams", [1, 2, 5])
def test_stream_join(streams):
    n, width, eps = 6, 10, 1e-2
    x, y = torch.randn(n, streams, width), torch.randn(n, width)
    a, b = randomise(HyperConnections(streams)), randomise(HyperConnections(streams))
    norm = randomise(RMSNorm(width, eps, offset=1.0))
    with torch.no_grad():
        got, h = a(x, SublayerResult(y), b.w_in, norm)
        want = plain.mix_streams(x.double(), y.double(), a.w_out.double(), a.mix.double())
        assert err(got, want) < TOL
        assert err(h, plain.norm_around_zero(plain.gather_streams(want, b.w_in.double()), norm.weight.double(), eps)) < TOL
        _, h = a(x, SublayerResult(y), None, norm, 0.3)   # the sum of the streams, scaled behind the norm
        assert err(h, 0.3 * plain.norm_around_zero(want.sum(1), norm.weight.double(), eps)) < TOL
        same, h = a(x, None, a.w_in, norm)                # nothing joins yet
        assert same is x and err(h, plain.norm_around_zero(plain.gather_streams(x.double(), a.w_in.double()), norm.weight.double(), eps)) < TOL


def test_mixers_alone():
    width, n, eps = 18, 21, 1e-3
    h = torch.randn(n, width)
    pos = torch.arange(n)[None]
    with torch.no_grad():
        m = attn(4, 2, 8, 0.4, 6, 2, 4, None, 100.0)["mixer"]
        a = randomise(GroupedQueryAttention(width, 4, 2, 8, 8, 0.4, eps, rot_dims=4, rot_base=100.0, norm_weights=False, sink=False, window=6,
                                            keep_first=2, value_is_key=True, gate="head"))
        get = getter({**{s: a.in_proj.part(s) for s in "qkg"}, "o": a.out_proj.weight})
        assert err(a(h, 1, 0, None, None, pos).y, plain.windowed_attention(h.double(), get, m, eps)) < TOL
        m = latent(3, 4, 6, 5, 7, 8, 0.3, None, 50.0)["mixer"]
        b = randomise(LatentAttention(width, 3, 4, 5, 7, 8, 0.3, eps, rot_dim=6, rot_base=50.0, sink=False, gate="element"))
        get = getter({"dq": b.in_proj.part("dq"), "dq.norm": b.q_norm.weight, "uq": b.uq.weight, "dkv": b.in_proj.part("dkv"), "dkv.norm": b.kv_norm.weight,
                      "uk": b.kv_up.part("k"), "uv": b.kv_up.part("v"), "g": b.in_proj.part("g"), "o": b.out_proj.weight})
        assert err(b(h, 1, 0, 0, None, None, None, False, pos).y, plain.latent_attention(h.double(), get, m, eps)) < TOL
        m = mlstm(3, 5, 4, 2.5, None)["mixer"]
        c = randomise(MatrixMemory(width, 3, 5, 4, 2.5, eps))
        get = getter({**{s: c.in_proj.part(s) for s in "qkvg"}, "i": c.gates.weight[:3], "f": c.gates.weight[3:], "i.b": c.gates.bias[:3],
                      "f.b": c.gates.bias[3:], "norm": c.o_norm, "o": c.out_proj.weight})
        assert err(c(h, 1, 0, None, None).y, plain.mlstm(h.double(), get, m, eps)[0]) < TOL
    with pytest.raises(ValueError):
        GroupedQueryAttention(width, 2, 1, 8, 6, 0.4, eps, value_is_key=True)
    with pytest.raises(ValueError):
        LatentAttention(width, 3, 4, 5, 7, 8, 0.3, eps, gate="row")
    with pytest.raises(ValueError):
        MixtureOfExperts(width, 4, 2, 1, unit="gelu")


def test_plain_states_carry_on():
    """The oracle itself: a recurrence in two pieces is the recurrence in one."""
    q, k, v = (torch.randn(9, 2, 3, dtype=torch.float64) for _ in range(3))
    i, f = torch.randn(9, 2, dtype=torch.float64), -torch.rand(9, 2, dtype=torch.float64)
    whole, end = plain.matrix_memory(q, k, v, i, f)
    first, state = plain.matrix_memory(q[:4], k[:4], v[:4], i[:4], f[:4])
    rest, last = plain.matrix_memory(q[4:], k[4:], v[4:], i[4:], f[4:], state)
    assert err(torch.cat([first, rest]), whole) < 1e-12 and all(err(a, b) < 1e-12 for a, b in zip(last, end))


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
    assert err(out.logits[0], want) < TOL and out.past_key_values is None
    assert [p is not None for p in out.attentions] == [l["type"] != "mlstm" for l in cfg["layers"]]


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
    assert float(d.median()) < 0.08                       # a close call of a router may go the other way at some positions


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
    # only what the design says is kept: keys and values of windowed layers, latents with the rotated part, matrix and maximum
    kinds = [l["type"] for l in cfg["layers"]]
    where = lambda kind: [i for i, k in enumerate(kinds) if k == kind]                          # noqa: E731
    assert sorted(cache.k) == where("attention") and sorted(cache.latent) == where("latent_attention")
    assert all(cache.latent[i].size(-1) == cfg["layers"][i]["mixer"]["kv_rank"] + cfg["layers"][i]["mixer"]["rot_dim"] for i in cache.latent)
    assert set(cache.state) == {k for i in where("mlstm") for k in (i, (i, "max"))}


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
    held = lambda c: sum(t.numel() for d in (c.k, c.v, c.latent, c.state) for t in d.values())  # noqa: E731
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


def test_keys_at_the_edges_of_a_window_count_or_do_not(tmp_path):
    """One windowed layer with even weights: changing a token changes exactly the positions that see it, in a prompt and in decoding."""
    size, kept, n = 20, 6, 70
    cfg = case(64, 40, 1e-5, 2, attn(2, 1, 16, 0.1, size, kept, 4, None, 1e5))
    model, tensors = load(tmp_path, cfg)
    seq = [t % 60 for t in ids(n, 60, 8)]
    want = plain.forward(cfg, tensors, seq)
    for prompt in (n, 45, 3):
        got = fed(model, seq, prompt)
        assert err(got, want) < 2 * TOL
        for at in (0, kept - 1, kept, kept + 1, 30, 44, 45):
            other = list(seq)
            other[at] = 61
            moved = (fed(model, other, prompt) - got).abs().amax(-1) / want.abs().max()
            for i in range(n):
                sees = plain.sees(i, at, size, kept)
                assert float(moved[i]) > 20 * TOL if sees else float(moved[i]) < TOL, (prompt, at, i)


def test_keys_far_away_decide_the_output_of_latent_attention(tmp_path):
    cfg = case(64, 40, 1e-5, 2, latent(2, 16, 8, 24, 24, 24, 0.5, None, 1e5), mlstm(1, 4, 4, 5.0, moe(8, 3, 1, 2, 8)))
    tensors = make_tensors(cfg, 3)
    for name in ("l0.mix.uq", "l0.mix.uk"):
        tensors[name] = tensors[name] * 2.0
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
        assert err(moved[max(at, 290):], want[max(at, 290):]) > 20 * TOL
        assert at == 0 or err(moved[:at], want[:at]) < 2 * TOL


def test_matrix_memory_carries_the_first_tokens_through_a_long_prompt(tmp_path):
    cfg = case(64, 24, 1e-5, 2, mlstm(2, 8, 12, 15.0, None), mlstm(1, 8, 8, 15.0, moe(16, 3, 1, 2, 16)))
    tensors = make_tensors(cfg, 4)
    for i in range(2):
        tensors[f"l{i}.mix.f.b"] = tensors[f"l{i}.mix.f.b"] * 0 + 14.0       # hardly forgets
        tensors[f"l{i}.mix.f"] = tensors[f"l{i}.mix.f"] * 0.1
    model, _ = load(tmp_path, cfg, tensors)
    seq = ids(260, 64, 9)
    want = plain.forward(cfg, tensors, seq)
    assert err(logits(model, seq)[0], want) < TOL and err(fed(model, seq, 100), want) < TOL
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
    x = torch.tensor([ids(40, 96, 14), ids(40, 96, 15)])
    mask = torch.ones_like(x)
    mask[1, :11] = 0
    model(input_ids=x, labels=x, attention_mask=mask).loss.backward()
    grads = {n: p.grad.clone() for n, p in model.named_parameters() if p.grad is not None}
    assert all(torch.isfinite(g).all() for g in grads.values())
    # corrections only choose: no gradient reaches them
    assert {n for n, p in model.named_parameters() if p.grad is None} == {n for n, _ in model.named_parameters() if n.endswith("mlp.correction")}
    assert all(g.abs().sum() > 0 for g in grads.values())
    model.zero_grad()
    model.gradient_checkpointing_enable()
    model(input_ids=x, labels=x, attention_mask=mask).loss.backward()
    for n, p in model.named_parameters():
        assert n not in grads or torch.allclose(p.grad, grads[n], atol=1e-5), n


def test_registry_and_loading(tmp_path):
    cfg = CASES["mixed"]
    tensors = make_tensors(cfg)
    model, _ = load(tmp_path / "a", cfg, tensors)
    assert type(model) is ob.DekutarForCausalLM and model.config.vocab_size == 96 and model.config.num_hidden_layers == 6
    model.save_pretrained(str(tmp_path / "b"))
    again = ob.load_causal_lm(str(tmp_path / "b"))
    seq = ids(8, 96)
    assert torch.equal(logits(again, seq), logits(model, seq))
    fresh = ob.DekutarForCausalLM(ob.DekutarConfig(**cfg))
    assert fresh(input_ids=torch.tensor([seq])).logits.isfinite().all()
    cls = ob.DekutarForSequenceClassification.from_pretrained(str(tmp_path / "b"))
    assert cls(input_ids=torch.tensor([seq])).logits.shape == (1, 2)
    for change, exc in ((lambda t: t.pop("l0.mix.k"), KeyError), (lambda t: t.update({"l9.x": torch.zeros(1)}), KeyError),
                        (lambda t: t.update({"l1.mix.o": torch.zeros(48, 33)}), ValueError), (lambda t: t.pop("l2.mlp.e3.gate"), KeyError),
                        (lambda t: t.update({"l2.mix.dkv": torch.zeros(41, 48)}), ValueError), (lambda t: t.pop("l1.hc2.mix"), KeyError)):
        t = dict(tensors)
        change(t)
        write_model(str(tmp_path / "c"), cfg, t)
        with pytest.raises(exc):
            ob.load_causal_lm(str(tmp_path / "c"))
    with pytest.raises(NotImplementedError):
        model._exec_both_engines(tensor_parallel_size=2)


def test_configurations_that_nothing_implements_are_refused():
    ob.DekutarConfig(**CASES["mixed"])
    without = lambda layer, key: {**layer, "mixer": {k: v for k, v in layer["mixer"].items() if k != key}}    # noqa: E731
    a, b, c = attn(2, 1, 8, 1.0, 4, 1, 4, None), latent(2, 8, 4, 8, 8, 8, 1.0, None), mlstm(1, 4, 4, 1.0, None)
    wide = {**a, "mixer": {**a["mixer"], "vdim": 16}}
    turned = {**b, "mixer": {**b["mixer"], "rot": {"dims": 2, "base": 10.0}}}
    for layer in ({"type": "window", "mixer": {}, "mlp": None}, attn(3, 2, 8, 1.0, 4, 1, 4, None), attn(2, 1, 8, 1.0, 4, 1, 10, None),
                  attn(2, 1, 8, 1.0, 0, 1, 4, None), attn(2, 1, 8, 1.0, 4, 1, 3, None), wide, turned, without(a, "mask"), without(b, "rot_dim"),
                  without(c, "gate_cap"), {**c, "mlp": {"kind": "dense", "ff": 3}}, {**c, "mlp": moe(4, 2, 1, 4, 4)}, {**c, "mlp": moe(4, 2, 1, 0, 4)}):
        with pytest.raises(ValueError):
            ob.DekutarConfig(layers=[layer], norm={"eps": 1e-5}, streams=2, vocab=8, width=8)
    for streams in (0, 17):
        with pytest.raises(ValueError):
            ob.DekutarConfig(layers=[c], streams=streams, vocab=8, width=8)


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
    cfg = case(256, 24, 1e-5, 2, mlstm(2, 8, 8, 9.0, moe(16, 3, 1, 2, 8)), attn(2, 1, 8, 0.4, 5, 2, 4, None), latent(2, 8, 4, 8, 12, 16, 0.3, None))
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
