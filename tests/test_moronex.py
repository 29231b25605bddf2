"""Moronex on the CPU statements of the ops: every mechanism against ``plain_moronex.py`` (double precision, loops), the cache and
the recurrent state under decoding, portions, padded batches, reordering and reuse, the scheduler and sampling paths of
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
from oslo_b200.models.mixers import GatedLinearRecurrence, GatedMLP, LatentAttention, MixtureOfExperts
from oslo_b200.parallel.layers import PackedLinear, RMSNorm

from . import plain_moronex as plain
from .moronex_cases import CASES, case, dense, far_key_weights, hgrn2, latent, make_tensors, moe, write_model

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


# ---------------------------------------------------------------------------------------------------- mechanisms alone
def test_rms_norms_put_eps_under_the_root():
    x = torch.randn(5, 24) * 1e-2
    w = torch.randn(24) * 0.3
    for offset, want in ((0.0, plain.norm_plain), (1.0, plain.norm_around_zero)):
        n = RMSNorm(24, 1e-2, offset)
        n.weight.data.copy_(w)
        assert err(n(x).detach(), want(x.double(), w.double(), 1e-2)) < TOL


def test_packed_linear_keeps_its_parts_apart_and_aligned():
    p = PackedLinear(12, {"a": 5, "b": 16, "c": 3})
    assert all(start % 8 == 0 for start, _ in p.parts.values()) and p.weight.shape == (8 + 16 + 8, 12)
    ws = {n: torch.randn(s, 12) for n, (_, s) in p.parts.items()}
    p.weight.data.copy_(p.pack(ws))
    x = torch.randn(4, 12)
    y = p(x)
    for n, w in ws.items():
        assert torch.equal(p.part(n), w) and err(y[n].detach(), x @ w.t()) < 1e-5
    with pytest.raises(KeyError):
        p.pack({"a": ws["a"]})
    with pytest.raises(ValueError):
        p.pack({**ws, "a": ws["b"]})


@pytest.mark.parametrize("heads,dim,vdim", [(1, 4, 6), (3, 10, 5), (2, 16, 16)])
def test_recurrence_is_the_token_by_token_rule(heads, dim, vdim):
    n = 11
    q, f = torch.randn(n, heads * dim), torch.randn(n, heads * dim)
    v, fb, lower = torch.randn(n, heads * vdim), torch.randn(heads * dim), torch.rand(heads * dim)
    s0 = torch.randn(1, heads, dim, vdim)
    gate = lower.double() + (1 - lower.double()) * plain.sigmoid(f.double() + fb.double())
    want, end = plain.linear_recurrence(plain.silu(q.double()).view(n, heads, dim), gate.view(n, heads, dim),
                                        v.double().view(n, heads, vdim), s0[0].double())
    got, state = ops.reference.recurrence(q, f, v, fb, lower, None, s0, 1, heads, dim, vdim)
    assert err(got[0], want) < TOL and err(state[0], end) < TOL
    # a padded token neither writes nor forgets, wherever it stands
    keep = torch.tensor([[1, 0, 1, 1, 0, 0, 1, 1, 1, 0, 1]])
    sel = keep[0].bool()
    want, end = plain.linear_recurrence(plain.silu(q.double()).view(n, heads, dim)[sel], gate.view(n, heads, dim)[sel],
                                        v.double().view(n, heads, vdim)[sel], s0[0].double())
    got, state = ops.reference.recurrence(q, f, v, fb, lower, keep, s0, 1, heads, dim, vdim)
    assert err(got[0][sel], want) < TOL and err(state[0], end) < TOL and not got[0][~sel].any()


def test_forget_gate_reaches_its_bounds():
    lower = torch.tensor([0.0, 0.5, 1.0])
    for z, want in ((-200.0, lower), (200.0, torch.ones(3))):
        s0 = torch.ones(1, 1, 3, 2)
        _, s = ops.reference.recurrence(torch.zeros(1, 3), torch.full((1, 3), z), torch.zeros(1, 2), torch.zeros(3), lower, None, s0,
                                        1, 1, 3, 2)
        assert torch.allclose(s[0, 0, :, 0], want)


def test_sink_counts_once_unscaled_and_without_a_value():
    n, heads, dim, vdim = 6, 3, 8, 5
    q, k, v = torch.randn(1, n, heads, dim), torch.randn(1, n, heads, dim), torch.randn(1, n, heads, vdim)
    sink, g = torch.tensor([-3.0, 0.0, 4.0]), torch.randn(n, heads)
    want = plain.sink_attention(q[0].double(), k[0].double(), v[0].double(), 0.7, sink.double()) * plain.sigmoid(g.double())[:, :, None]
    got, probs = ops.reference.sink_attention(q, k, v, None, sink, g, 0.7)
    assert err(got.view(n, heads, vdim), want) < TOL
    # the first token sees itself and the sink only
    e = math.exp(float((q[0, 0, 2] @ k[0, 0, 2]) * 0.7))
    assert abs(float(probs[0, 2, 0, 0]) - e / (e + math.exp(4.0))) < 1e-5
    # the last queries of a longer sequence, and a far key that stands out
    k[0, 0, 1] = 4.0 * q[0, 5, 1]
    full, _ = ops.reference.sink_attention(q, k, v, None, sink, g, 0.7)
    tail, p = ops.reference.sink_attention(q[:, 4:], k, v, None, sink, g[4:], 0.7)
    assert err(tail, full[4:]) < 1e-6 and float(p[0, 1, 1, 0]) > 0.9


@pytest.mark.parametrize("rank,heads,dim,vdim", [(12, 2, 8, 6), (20, 3, 5, 16)])
def test_latent_attention_expanded_and_absorbed(rank, heads, dim, vdim):
    width, q_rank, n, eps = 18, 14, 9, 1e-4
    m = LatentAttention(width, heads, dim, vdim, q_rank, rank, 0.4, eps)
    for p in m.parameters():
        p.data.normal_(std=0.5)
    get = {"dq": m.in_proj.part("dq"), "dq.norm": m.q_norm.weight, "uq": m.uq.weight, "dkv": m.in_proj.part("dkv"),
           "dkv.norm": m.kv_norm.weight, "uk": m.kv_up.part("k"), "uv": m.kv_up.part("v"), "sink": m.sink,
           "g": m.in_proj.part("g"), "o": m.out_proj.weight}
    get = {k: v.detach().double() for k, v in get.items()}
    h = torch.randn(n, width)
    c = plain.latents(h.double(), get.__getitem__, eps)
    want = plain.latent_attention(h.double(), c, get.__getitem__, dict(heads=heads, dim=dim, vdim=vdim, scale=0.4), eps)
    with torch.no_grad():
        out = m(h, 1, 0, 0, None, None, None)
        assert err(out.y, want) < TOL and err(out.latent[0], c) < TOL
        # the decode form on the same latents
        p = m.in_proj(h)
        q = m.uq(m.q_norm(p["dq"]))
        cache = torch.zeros(1, 13, rank)
        cache[0, :n] = out.latent[0]
        o = ops.latent_decode(q[-1:], get["uk"].float(), get["uv"].float(), cache, torch.tensor([n]), None, m.sink, p["g"][-1:], 0.4, heads)
        assert err(m.out_proj(o), want[-1:]) < TOL


def test_router_weights_are_the_softmax_over_the_chosen_logits():
    h, w, b = torch.randn(40, 10), torch.randn(7, 10), torch.randn(7)
    for top in (1, 3, 7):
        idx, wgt = ops.reference.moe_route(h, w, b, top)
        pi, pw = plain.route(h.double(), w.double(), b.double(), top)
        assert torch.equal(idx.long(), pi) and err(wgt, pw) < TOL


def test_feed_forwards():
    h = torch.randn(9, 12)
    d = GatedMLP(12, 20)
    get = {"gate": d.in_proj.part("gate"), "up": d.in_proj.part("up"), "down": d.down.weight}
    get = {k: v.detach().double() for k, v in get.items()}
    assert err(d(h).y.detach(), plain.dense_mlp(h.double(), get.__getitem__)) < TOL
    m = MixtureOfExperts(12, 6, 5, 2)
    m.up.data.normal_(); m.down.data.normal_(); m.router.weight.data.normal_()
    get = {"router": m.router.weight, "router.b": m.router.bias}
    for e in range(5):
        get[f"e{e}.up"], get[f"e{e}.down"] = m.up[e], m.down[e]
    get = {k: v.detach().double() for k, v in get.items()}
    f = m(h)
    got = (f.y.view(9, 2, 12) * f.weights.unsqueeze(-1)).sum(1)
    assert err(got.detach(), plain.moe_mlp(h.double(), get.__getitem__, {"top": 2})) < TOL


def test_residual_join_gates_then_norms_then_adds():
    x, y, g, b = torch.randn(6, 10), torch.randn(6, 10), torch.randn(6, 10), torch.randn(10)
    wp, wn = torch.randn(10), torch.randn(10)
    want = x.double() + plain.norm_around_zero(y.double() * plain.sigmoid(g.double() + b.double()), wp.double(), 1e-3)
    got, h = ops.reference.residual_join(x, y, g, b, wp, wn, 1e-3)
    assert err(got, want) < TOL and err(h, plain.norm_around_zero(want, wn.double(), 1e-3)) < TOL


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


@pytest.mark.parametrize("name", sorted(CASES))
def test_sixteen_bit_model_keeps_the_stream_in_32_bit(tmp_path, name):
    cfg = CASES[name]
    model, tensors = load(tmp_path, cfg, dtype=torch.bfloat16)
    seq = ids(20, cfg["vocab"])
    with torch.no_grad():
        out = model(input_ids=torch.tensor([seq]), output_hidden_states=True)
    assert all(h.dtype == torch.float32 for h in out.hidden_states)
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
    # only what the design says is kept: one latent per token and own-latent layer, one state per recurrent layer
    own = [i for i, l in enumerate(cfg["layers"]) if l["type"] == "latent_attention" and "kv_from" not in l["mixer"]]
    rec = [i for i, l in enumerate(cfg["layers"]) if l["type"] == "hgrn2"]
    assert sorted(cache.latent) == own and sorted(cache.state) == rec and not cache.k and not cache.v
    assert all(s.dtype == torch.float32 for s in cache.state.values())


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
    cache = steps.kwargs["past_key_values"]
    before = sum(t.numel() for d in (cache.latent, cache.state) for t in d.values())
    steps.keep([1])
    cache = steps.kwargs["past_key_values"]
    assert sum(t.numel() for d in (cache.latent, cache.state) for t in d.values()) * 2 == before
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


def test_cache_limits():
    cache = StaticKVCache(4)
    cache.append_latent(0, torch.ones(1, 3, 2))
    cache.advance(3)
    with pytest.raises(RuntimeError, match="overflow"):
        cache.append_latent(0, torch.ones(1, 2, 2))
    grow = StaticKVCache(4, grow=True)
    for i in range(9):
        c = grow.append_latent(0, torch.full((2, 1, 2), float(i)))
        grow.advance(1)
    assert c.shape == (2, 9, 2) and torch.equal(c[1, :, 0], torch.arange(9.0)) and int(grow.lengths_dev[1]) == 9


def test_keys_far_away_decide_the_output(tmp_path):
    """With attention sharpened to a search, a prompt's and a decoded token's result hang on single keys hundreds of tokens
    back: changing such a key's token changes the logits, and all ways of feeding the sequence agree with the plain model."""
    cfg = case(64, 40, 1e-5, latent(2, 16, 24, 32, 24, 1.0, None), latent(2, 16, 24, 32, 24, 1.0, None, kv_from=0),
               hgrn2(2, 8, 16, dense(24)))
    tensors = far_key_weights(cfg, 0, make_tensors(cfg, 3))
    model, _ = load(tmp_path, cfg, tensors)
    seq = [t % 60 for t in ids(300, 60, 8)]
    for at in (0, 1, 150):
        seq[at] = 63                                      # a rare token: a key of its own
    want = plain.forward(cfg, tensors, seq)
    assert err(logits(model, seq)[0], want) < TOL
    cache = StaticKVCache(320)
    with torch.no_grad():
        model(input_ids=torch.tensor([seq[:290]]), past_key_values=cache)
        got = torch.cat([model(input_ids=torch.tensor([[t]]), past_key_values=cache).logits[0] for t in seq[290:]])
    assert err(got, want[290:]) < TOL
    for at in (0, 1, 150):
        other = list(seq)
        other[at] = 62
        moved = logits(model, other)[0]
        assert err(moved[max(at, 290):], want[max(at, 290):]) > 20 * TOL
        assert at == 0 or err(moved[:at], want[:at]) < TOL


def test_recurrent_state_carries_the_first_tokens_through_a_long_prompt(tmp_path):
    cfg = case(64, 24, 1e-5, hgrn2(2, 12, 8, None), hgrn2(1, 8, 16, dense(16)))
    tensors = make_tensors(cfg, 4)
    for i in range(2):
        tensors[f"l{i}.mix.f.b"] = tensors[f"l{i}.mix.f.b"] + 5.0          # hardly forgets
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
    want = torch.tensor([plain_greedy(cfg, tensors, p, 12) for p in prompts])
    kw = dict(max_new_tokens=12, eos_token_id=None, pad_token_id=None)
    assert torch.equal(model.generate(torch.tensor(prompts), **kw), want)
    assert torch.equal(model.generate(torch.tensor(prompts), use_static_cache=False, **kw), want)
    dec = GraphedGreedyDecoder(model, max_len=40, use_graph=False)
    for _ in range(2):                                    # the decoder's cache and state are reused
        assert torch.equal(dec.generate(torch.tensor(prompts), 12), want)
    # unequal prompts, padded on the left
    short = prompts[1][:4]
    padded = torch.tensor([prompts[0], [0] * 5 + short])
    mask = torch.tensor([[1] * 9, [0] * 5 + [1] * 4])
    got = model.generate(padded, attention_mask=mask, **kw)
    assert got[0].tolist() == want[0].tolist() and got[1, 5:].tolist() == plain_greedy(cfg, tensors, short, 12)


def test_sampling_and_beam_search(tmp_path):
    cfg = CASES["mixed"]
    model, _ = load(tmp_path, cfg)
    x = torch.tensor([ids(6, 96, 13)])
    torch.manual_seed(0)
    a = model.generate(x, do_sample=True, top_k=5, max_new_tokens=8, num_return_sequences=3, eos_token_id=None, pad_token_id=0)
    assert a.shape == (3, 14)
    got = model.generate(x, num_beams=3, max_new_tokens=8, eos_token_id=None, pad_token_id=0, return_dict_in_generate=True)
    # the best beam's score is what the model gives that sequence
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
    assert all(torch.isfinite(g).all() for g in grads.values()) and all(g.abs().sum() > 0 for n, g in grads.items() if "experts" not in n)
    model.zero_grad()
    model.gradient_checkpointing_enable()
    model(input_ids=x, labels=x).loss.backward()
    for n, p in model.named_parameters():
        assert torch.allclose(p.grad, grads[n], atol=1e-6), n


def test_registry_and_loading(tmp_path):
    cfg = CASES["mixed"]
    tensors = make_tensors(cfg)
    model, _ = load(tmp_path / "a", cfg, tensors)
    assert type(model) is ob.MoronexForCausalLM and model.config.vocab_size == 96 and model.config.num_hidden_layers == 4
    model.save_pretrained(str(tmp_path / "b"))
    again = ob.load_causal_lm(str(tmp_path / "b"))
    seq = ids(8, 96)
    assert torch.equal(logits(again, seq), logits(model, seq))
    assert ob.find_model({"architectures": ["GPTJForCausalLM"]}).causal_lm is ob.GPTJForCausalLM
    assert ob.find_model({"model_type": "gpt2"}).config is ob.GPT2Config
    with pytest.raises(ValueError):
        ob.find_model({"architecture": "Nothing"})
    cls = ob.MoronexForSequenceClassification.from_pretrained(str(tmp_path / "b"))
    assert cls(input_ids=torch.tensor([seq])).logits.shape == (1, 2)
    for change, exc in ((lambda t: t.pop("l2.mix.uk"), KeyError), (lambda t: t.update({"l9.x": torch.zeros(1)}), KeyError),
                        (lambda t: t.update({"l1.mix.o": torch.zeros(48, 33)}), ValueError)):
        t = dict(tensors)
        change(t)
        write_model(str(tmp_path / "c"), cfg, t)
        with pytest.raises(exc):
            ob.load_causal_lm(str(tmp_path / "c"))
    with pytest.raises(NotImplementedError):
        model._exec_both_engines(tensor_parallel_size=2)


def test_configurations_that_nothing_implements_are_refused():
    good = CASES["mixed"]["layers"]
    ob.MoronexConfig(layers=good, norm={"eps": 1e-5}, vocab=8, width=8)
    for layers in ([{"type": "window", "mixer": {}, "mlp": None}], [latent(1, 4, 4, 4, 4, 1.0, None, kv_from=0)],
                   [latent(1, 4, 4, 4, 4, 1.0, None), latent(1, 4, 4, 4, 8, 1.0, None, kv_from=0)],
                   [latent(1, 4, 4, 4, 4, 1.0, None), latent(1, 4, 4, 4, 4, 1.0, None, kv_from=0), latent(1, 4, 4, 4, 4, 1.0, None, kv_from=1)],
                   [hgrn2(1, 4, 4, moe(4, 2, 3))], [hgrn2(1, 4, 4, {"kind": "other"})], [{"type": "hgrn2", "mixer": {"heads": 1}, "mlp": None}]):
        with pytest.raises(ValueError):
            ob.MoronexConfig(layers=layers, norm={"eps": 1e-5}, vocab=8, width=8)


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
    from oslo_b200.trace import TraceRunner
    r = TraceRunner(model, str(out))
    r.step(lines[0])
    with pytest.raises(ValueError):                       # nobody joins a batch that has started
        r.step({"step": 1, "entries": [{"id": "a", "tokens": a[7:8]}, {"id": "new", "tokens": [1]}], "end": []})
    with pytest.raises(ValueError):
        r.step({"step": 1, "entries": [{"id": "a", "tokens": a[7:9]}], "end": []})


def test_generate_command_line(tmp_path):
    cfg = case(256, 24, 1e-5, hgrn2(2, 8, 12, moe(16, 3, 2)), latent(2, 8, 12, 16, 16, 0.3, dense(32)))
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
