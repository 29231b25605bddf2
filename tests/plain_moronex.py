"""A plain, slow Moronex in double precision: one function per mechanism, loops where a loop is the definition.

It works on a nested configuration dictionary and a flat ``{tensor name: tensor}`` dictionary, one unpadded sequence at a
time, and imports nothing from the package: the tests compare the package against it. ``x`` is always ``[tokens, width]``.
"""
import math

import torch

F64 = torch.float64


def silu(z):
    return z / (1.0 + torch.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def rms(x, eps):
    """Rows divided by their root mean square, eps under the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_zero(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def norm_plain(x, w, eps):
    return rms(x, eps) * w


def residual_gate(h, w, b):
    return sigmoid(h @ w.T + b)


def forget_gate(h, w_f, b_f, lower):
    """``[tokens, heads * dim]``, between ``lower`` and 1."""
    return lower + (1.0 - lower) * sigmoid(h @ w_f.T + b_f)


def linear_recurrence(q, f, v, state=None):
    """``q, f [tokens, heads, dim]``, ``v [tokens, heads, vdim]``: token by token, head by head. Returns the outputs
    ``[tokens, heads, vdim]`` and the state ``[heads, dim, vdim]`` after the last token."""
    tokens, heads, dim = q.shape
    vdim = v.shape[-1]
    s = torch.zeros(heads, dim, vdim, dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros(tokens, heads, vdim, dtype=q.dtype)
    for t in range(tokens):
        for a in range(heads):
            s[a] = f[t, a][:, None] * s[a] + (1.0 - f[t, a])[:, None] * v[t, a][None, :]
            out[t, a] = s[a].T @ q[t, a]
    return out, s


def hgrn2(h, get, m, eps, state=None):
    heads, dim, vdim = m["heads"], m["dim"], m["vdim"]
    n = h.shape[0]
    q = silu(h @ get("q").T).reshape(n, heads, dim)
    f = forget_gate(h, get("f"), get("f.b"), get("lower")).reshape(n, heads, dim)
    v = (h @ get("v").T).reshape(n, heads, vdim)
    o, state = linear_recurrence(q, f, v, state)
    o = norm_plain(o, get("norm"), eps)
    return o.reshape(n, heads * vdim) @ get("o").T, state


def sink_attention(q, k, v, scale, sink):
    """``q [n, heads, dim]`` are the last ``n`` of the positions that ``k [t, heads, dim]`` / ``v`` cover; causal softmax whose
    denominator also holds ``exp(sink[head])``."""
    n, heads, _ = q.shape
    t = k.shape[0]
    out = torch.zeros(n, heads, v.shape[-1], dtype=q.dtype)
    for i in range(n):
        last = t - n + i
        for a in range(heads):
            s = (k[:last + 1, a] @ q[i, a]) * scale
            top = max(float(s.max()), float(sink[a]))
            e = torch.exp(s - top)
            out[i, a] = (e @ v[:last + 1, a]) / (e.sum() + math.exp(float(sink[a]) - top))
    return out


def latents(h, get, eps):
    return norm_plain(h @ get("dkv").T, get("dkv.norm"), eps)


def latent_attention(h, c, get, m, eps):
    """``h`` are the last rows of the sequence whose latents are ``c``."""
    heads, dim, vdim = m["heads"], m["dim"], m["vdim"]
    n, t = h.shape[0], c.shape[0]
    q = (norm_plain(h @ get("dq").T, get("dq.norm"), eps) @ get("uq").T).reshape(n, heads, dim)
    k = (c @ get("uk").T).reshape(t, heads, dim)
    v = (c @ get("uv").T).reshape(t, heads, vdim)
    o = sink_attention(q, k, v, m["scale"], get("sink"))
    o = o * sigmoid(h @ get("g").T)[:, :, None]
    return o.reshape(n, heads * vdim) @ get("o").T


def dense_mlp(h, get):
    return (silu(h @ get("gate").T) * (h @ get("up").T)) @ get("down").T


def route(h, w, b, top):
    """Per token the chosen experts and their weights."""
    z = h @ w.T + b
    chosen = torch.sort(z, dim=-1, descending=True, stable=True).indices[:, :top]
    picked = torch.gather(z, 1, chosen)
    e = torch.exp(picked - picked.max(-1, keepdim=True).values)
    return chosen, e / e.sum(-1, keepdim=True)


def moe_mlp(h, get, r):
    chosen, weight = route(h, get("router"), get("router.b"), r["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(r["top"]):
            e = int(chosen[t, j])
            a = torch.clamp(get(f"e{e}.up") @ h[t], min=0.0) ** 2
            out[t] += weight[t, j] * (get(f"e{e}.down") @ a)
    return out


def forward(cfg, tensors, tokens, keep_layers=False):
    """Logits ``[tokens, vocab]`` of one sequence (and the residual stream after every layer)."""
    p = {k: v.to(F64) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = p["embed"][torch.as_tensor(tokens)]
    stream, caches = [], {}
    for i, layer in enumerate(cfg["layers"]):
        get = lambda name, i=i: p[f"l{i}.mix.{name}"]                                   # noqa: E731
        m = layer["mixer"]
        h = norm_around_zero(x, p[f"l{i}.norm1"], eps)
        if layer["type"] == "hgrn2":
            y, _ = hgrn2(h, get, m, eps)
        else:
            if m.get("kv_from") is None:
                caches[i] = latents(h, get, eps)
            y = latent_attention(h, caches[i if m.get("kv_from") is None else m["kv_from"]], get, m, eps)
        y = y * residual_gate(h, p[f"l{i}.rg1"], p[f"l{i}.rg1.b"])
        x = x + norm_around_zero(y, p[f"l{i}.norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            get = lambda name, i=i: p[f"l{i}.mlp.{name}"]                               # noqa: E731
            h = norm_around_zero(x, p[f"l{i}.norm2"], eps)
            y = dense_mlp(h, get) if mlp["kind"] == "dense" else moe_mlp(h, get, mlp["router"])
            y = y * residual_gate(h, p[f"l{i}.rg2"], p[f"l{i}.rg2.b"])
            x = x + norm_around_zero(y, p[f"l{i}.norm2b"], eps)
        stream.append(x)
    logits = norm_around_zero(x, p["final.norm"], eps) @ p["head"].T
    return (logits, torch.stack(stream)) if keep_layers else logits
