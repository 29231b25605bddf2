"""A plain, slow Begovik in double precision: one function per mechanism, loops where a loop is the definition.

It works on a nested configuration dictionary and a flat ``{tensor name: tensor}`` dictionary, one unpadded sequence at a
time, and imports nothing from the package: the tests compare the package against it. ``x`` and ``h`` are ``[tokens, width]``.
"""
import math

import torch

F64 = torch.float64


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def rms(x, eps):
    """Rows divided by their root mean square, eps under the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return rms(x, eps) * w


# ------------------------------------------------------------------------------------------ grouped-query attention
def rotate(x, dims, base):
    """``x [tokens, heads, dim]``: pairs ``(2i, 2i + 1)`` of the first ``dims`` dimensions turn by ``position * base^(-2i / dims)``."""
    out = x.clone()
    for i in range(dims // 2):
        a = torch.arange(x.shape[0], dtype=x.dtype) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i] = u * c - v * s
        out[:, :, 2 * i + 1] = v * c + u * s
    return out


def soften(s, cap):
    return cap * torch.tanh(s / cap)


def capped_attention(q, k, v, scale, cap):
    """``q [n, H, dim]`` are the last ``n`` positions of ``k [t, G, dim]`` / ``v [t, G, vdim]``; query head ``h`` reads group
    ``h // (H / G)``; the denominator also holds ``exp(0)``."""
    n, heads, _ = q.shape
    t, groups, vdim = v.shape
    out = torch.zeros(n, heads, vdim, dtype=q.dtype)
    for i in range(n):
        last = t - n + i
        for a in range(heads):
            g = a // (heads // groups)
            s = soften((k[:last + 1, g] @ q[i, a]) * scale, cap)
            top = max(float(s.max()), 0.0)
            e = torch.exp(s - top)
            out[i, a] = (e @ v[:last + 1, g]) / (e.sum() + math.exp(-top))
    return out


def attention(h, get, m, eps):
    n, heads, groups, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = norm((h @ get("q").T).reshape(n, heads, dim), get("q.norm"), eps)
    k = norm((h @ get("k").T).reshape(n, groups, dim), get("k.norm"), eps)
    v = (h @ get("v").T).reshape(n, groups, vdim)
    q, k = (rotate(t, m["rot"]["dims"], m["rot"]["base"]) for t in (q, k))
    return capped_attention(q, k, v, m["scale"], m["softcap"]).reshape(n, heads * vdim) @ get("o").T


# ------------------------------------------------------------------------------------------ constant decay
def decayed_sum(q, k, v, decay, state=None):
    """``q, k [tokens, heads, dim]``, ``v [tokens, heads, vdim]``, ``decay [heads]``: a token is written, then read."""
    n, heads, dim = q.shape
    s = torch.zeros(heads, dim, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros(n, heads, v.shape[-1], dtype=q.dtype)
    for t in range(n):
        for a in range(heads):
            s[a] = decay[a] * s[a] + k[t, a][:, None] * v[t, a][None, :]
            out[t, a] = s[a].T @ q[t, a]
    return out, s


def lightning(h, get, m, eps, state=None):
    n, heads, dim, vdim = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(h @ get("q").T).reshape(n, heads, dim)
    k = silu(h @ get("k").T).reshape(n, heads, dim)
    v = silu(h @ get("v").T).reshape(n, heads, vdim)
    o, state = decayed_sum(q, k, v, torch.tensor(m["decay"], dtype=h.dtype), state)
    o = norm(o.reshape(n, heads * vdim), get("norm"), eps) * sigmoid(h @ get("g").T)
    return o @ get("o").T, state


def parallel(h, get, m, eps):
    left = attention(h, lambda name: get("left." + name), m["left"], eps)
    right, _ = lightning(h, lambda name: get("right." + name), m["right"], eps)
    return 0.5 * (norm(left, get("left.out"), eps) + norm(right, get("right.out"), eps))


# ------------------------------------------------------------------------------------------ wkv
def shifted(h, before=None):
    """The row before each row; ``before`` (zeros at the start of a sequence) is the one before the first."""
    first = torch.zeros(1, h.shape[1], dtype=h.dtype) if before is None else before[None]
    return torch.cat([first, h[:-1]])


def channel_decay(mix_w, w1, w2, w0):
    """``[tokens, heads * dim]``, between 0 and 1."""
    return torch.exp(-torch.exp(torch.tanh(mix_w @ w1.T) @ w2.T + w0))


def bonus_recurrence(r, k, v, w, u, state=None):
    """All ``[tokens, heads, dim]``, ``u [heads, dim]``: a token is read with the bonus, the state with the tokens before it."""
    n, heads, dim = r.shape
    s = torch.zeros(heads, dim, dim, dtype=r.dtype) if state is None else state.clone()
    out = torch.zeros(n, heads, dim, dtype=r.dtype)
    for t in range(n):
        for a in range(heads):
            kv = k[t, a][:, None] * v[t, a][None, :]
            out[t, a] = (s[a] + u[a][:, None] * kv).T @ r[t, a]
            s[a] = w[t, a][:, None] * s[a] + kv
    return out, s


def wkv(h, get, m, eps, before=None, state=None):
    n, heads, dim = h.shape[0], m["heads"], m["dim"]
    prev = shifted(h, before)
    mix = {s: h + (prev - h) * get("mu." + s) for s in "rkvgw"}
    r, k, v = ((mix[s] @ get(s).T).reshape(n, heads, dim) for s in "rkv")
    gate = silu(mix["g"] @ get("g").T)
    w = channel_decay(mix["w"], get("w1"), get("w2"), get("w0")).reshape(n, heads, dim)
    o, state = bonus_recurrence(r, k, v, w, get("u").reshape(heads, dim), state)
    o = rms(o, eps).reshape(n, heads * dim) * get("norm") * gate
    return o @ get("o").T, state


# ------------------------------------------------------------------------------------------ selective scan
def causal_conv(x, taps, bias, before=None):
    """``x [tokens, channels]``, ``taps [channels, n]`` with the current token's last; ``before``: the ``n - 1`` rows ahead of ``x``."""
    n = taps.shape[1]
    pad = torch.zeros(n - 1, x.shape[1], dtype=x.dtype) if before is None else before
    full = torch.cat([pad, x])
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(n):
            out[t] += taps[:, j] * full[t + j]
        out[t] += bias
    return out


def selective_scan(x, dt, a, b, c, d, state=None):
    """``x, dt [tokens, channels]``, ``a [channels, n]`` (negative), ``b, c [tokens, n]``, ``d [channels]``."""
    s = torch.zeros_like(a) if state is None else state.clone()
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        s = torch.exp(dt[t][:, None] * a) * s + (dt[t] * x[t])[:, None] * b[t][None, :]
        out[t] = s @ c[t] + d * x[t]
    return out, s


def mamba1(h, get, m, eps, state=None):
    inner, rank, n = m["inner"], m["dt_rank"], m["state"]
    x, z = (h @ get("in").T).split([inner, inner], dim=-1)
    x = silu(causal_conv(x, get("conv"), get("conv.b")))
    dt, b, c = (x @ get("x").T).split([rank, n, n], dim=-1)
    dt = softplus(dt @ get("dt").T + get("dt.b"))
    y, state = selective_scan(x, dt, -torch.exp(get("A_log")), b, c, get("D"), state)
    return (y * silu(z)) @ get("o").T, state


# ------------------------------------------------------------------------------------------ feed-forward, model
def clamped_glu(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def dense_mlp(h, get, limit):
    return clamped_glu(h @ get("gate").T, h @ get("up").T, limit) @ get("down").T


MIXERS = {"parallel": lambda *a: (parallel(*a), None), "wkv": wkv, "mamba1": mamba1}


def forward(cfg, tensors, tokens, keep_layers=False):
    """Logits ``[tokens, vocab]`` of one sequence (and the residual stream after every layer)."""
    p = {k: v.to(F64) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = p["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    stream = []
    for i, layer in enumerate(cfg["layers"]):
        get = lambda name, i=i: p[f"l{i}.mix.{name}"]                                   # noqa: E731
        y, _ = MIXERS[layer["type"]](norm(x, p[f"l{i}.norm1"], eps), get, layer["mixer"], eps)
        if layer.get("mlp") is not None:
            get = lambda name, i=i: p[f"l{i}.mlp.{name}"]                               # noqa: E731
            y = y + dense_mlp(norm(x, p[f"l{i}.norm2"], eps), get, layer["mlp"]["limit"])
        x = x + cfg["residual_mult"] * y
        stream.append(x)
    logits = norm(x, p["final.norm"], eps) @ p["head"].T
    return (logits, torch.stack(stream)) if keep_layers else logits
