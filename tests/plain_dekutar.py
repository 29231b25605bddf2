"""A plain, slow Dekutar in double precision: one function per mechanism, loops where a loop is the definition.

It works on a nested configuration dictionary and a flat ``{tensor name: tensor}`` dictionary, one unpadded sequence at a
time, and imports nothing from the package: the tests compare the package against it. ``h`` is ``[tokens, width]``, the
residual streams are ``[tokens, streams, width]``.
"""
import math

import torch

F64 = torch.float64


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def log_sigmoid(z):
    return torch.clamp(z, max=0.0) - torch.log1p(torch.exp(-z.abs()))


def rms(x, eps):
    """Rows divided by their root mean square, eps under the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_plain(x, w, eps):
    return rms(x, eps) * w


def norm_around_zero(x, w, eps):
    return rms(x, eps) * (1.0 + w)


# ------------------------------------------------------------------------------------------ residual streams
def gather_streams(x, w_in):
    """What a sublayer reads: ``[tokens, width]``."""
    out = torch.zeros_like(x[:, 0])
    for s in range(x.shape[1]):
        out += w_in[s] * x[:, s]
    return out


def mix_streams(x, y, w_out, mix):
    """The streams after a sublayer's result ``y``; ``mix [from, to]``."""
    out = torch.zeros_like(x)
    for t in range(x.shape[1]):
        for s in range(x.shape[1]):
            out[:, t] += mix[s, t] * x[:, s]
        out[:, t] += w_out[t] * y
    return out


# ------------------------------------------------------------------------------------------ rotation
def angle(position, i, dims, base):
    return position * base ** (-2.0 * i / dims)


def rotate_pairs(x, pairs, dims, base, first=0):
    """``x [tokens, heads, dim]``, the first token at position ``first``; ``pairs(i)`` are the two dimensions of pair ``i``."""
    out = x.clone()
    for t in range(x.shape[0]):
        for i in range(dims // 2):
            a = angle(first + t, i, dims, base)
            c, s = math.cos(a), math.sin(a)
            p, q = pairs(i)
            out[t, :, p] = x[t, :, p] * c - x[t, :, q] * s
            out[t, :, q] = x[t, :, q] * c + x[t, :, p] * s
    return out


def rotate_interleaved(x, dims, base, first=0):
    return rotate_pairs(x, lambda i: (2 * i, 2 * i + 1), dims, base, first)


def rotate_halves(x, dims, base, first=0):
    return rotate_pairs(x, lambda i: (i, i + dims // 2), dims, base, first)


# ------------------------------------------------------------------------------------------ attention
def sees(i, j, size=None, keep_first=0):
    """Whether position ``i`` reads position ``j``; ``size`` ``None``: no window."""
    return j <= i and (size is None or i - j < size or j < keep_first)


def softmax_attention(q, k, v, scale, size=None, keep_first=0):
    """``q [n, H, dim]`` are the last ``n`` positions of ``k [t, G, dim]`` / ``v [t, G, vdim]``; query head ``h`` reads group
    ``h // (H / G)``."""
    n, heads, _ = q.shape
    t, groups, vdim = v.shape
    out = torch.zeros(n, heads, vdim, dtype=q.dtype)
    for i in range(n):
        at = [j for j in range(t) if sees(t - n + i, j, size, keep_first)]
        for a in range(heads):
            g = a // (heads // groups)
            s = (k[at, g] @ q[i, a]) * scale
            e = torch.exp(s - s.max())
            out[i, a] = (e @ v[at, g]) / e.sum()
    return out


def windowed_attention(h, get, m, eps):
    n, heads, groups, dim = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    rot, mask = m["rot"], m["mask"]
    q = (h @ get("q").T).reshape(n, heads, dim)
    k = (h @ get("k").T).reshape(n, groups, dim)
    v = k
    q, k = (rms(rotate_interleaved(t, rot["dims"], rot["base"]), eps) for t in (q, k))
    o = softmax_attention(q, k, v, m["scale"], mask["size"], mask["keep_first"])
    o = o * sigmoid(h @ get("g").T)[:, :, None]
    return o.reshape(n, -1) @ get("o").T


def latent_attention(h, get, m, eps):
    n, heads, dim, rot, rank, vdim = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"], m["vdim"]
    base = m["rot"]["base"]
    q = (norm_plain(h @ get("dq").T, get("dq.norm"), eps) @ get("uq").T).reshape(n, heads, dim + rot)
    both = h @ get("dkv").T
    c = norm_plain(both[:, :rank], get("dkv.norm"), eps)
    shared = rotate_halves(both[:, None, rank:], rot, base)
    q = torch.cat([q[:, :, :dim], rotate_halves(q[:, :, dim:], rot, base)], dim=-1)
    k = torch.cat([(c @ get("uk").T).reshape(n, heads, dim), shared.expand(n, heads, rot)], dim=-1)
    v = (c @ get("uv").T).reshape(n, heads, vdim)
    o = softmax_attention(q, k, v, m["scale"]).reshape(n, heads * vdim)
    return (o * sigmoid(h @ get("g").T)) @ get("o").T


# ------------------------------------------------------------------------------------------ matrix memory
def capped(z, cap):
    return cap * torch.tanh(z / cap)


def matrix_memory(q, k, v, i, f, state=None):
    """``q, k [tokens, heads, dim]``, ``v [tokens, heads, vdim]``, log gates ``i, f [tokens, heads]``. State: the matrices
    ``[heads, dim, vdim]``, the normalisers ``[heads, dim]`` and the running maxima ``[heads]``."""
    n, heads, dim = q.shape
    if state is None:
        state = (torch.zeros(heads, dim, v.shape[-1], dtype=q.dtype), torch.zeros(heads, dim, dtype=q.dtype),
                 torch.zeros(heads, dtype=q.dtype))
    s, z, m = (t.clone() for t in state)
    out = torch.zeros(n, heads, v.shape[-1], dtype=q.dtype)
    for t in range(n):
        for a in range(heads):
            new = max(float(f[t, a] + m[a]), float(i[t, a]))
            forget, write = math.exp(float(f[t, a] + m[a]) - new), math.exp(float(i[t, a]) - new)
            s[a] = forget * s[a] + write * k[t, a][:, None] * v[t, a][None, :]
            z[a] = forget * z[a] + write * k[t, a]
            m[a] = new
            out[t, a] = (s[a].T @ q[t, a]) / (max(abs(float(z[a] @ q[t, a])), math.exp(-new)) + 1e-6)
    return out, (s, z, m)


def mlstm(h, get, m, eps, state=None):
    n, heads, dim, vdim, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ get("q").T).reshape(n, heads, dim) * dim ** -0.5
    k = (h @ get("k").T).reshape(n, heads, dim)
    v = (h @ get("v").T).reshape(n, heads, vdim)
    i = capped(h @ get("i").T + get("i.b"), cap)
    f = log_sigmoid(capped(h @ get("f").T + get("f.b"), cap))
    o, state = matrix_memory(q, k, v, i, f, state)
    o = rms(o, eps).reshape(n, heads * vdim) * get("norm") * sigmoid(h @ get("g").T)
    return o @ get("o").T, state


# ------------------------------------------------------------------------------------------ feed-forward
def gated_unit(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def route(h, w, correction, top):
    """Per token the chosen outputs and their weights."""
    z = h @ w.T
    e = torch.exp(z - z.max(-1, keepdim=True).values)
    s = e / e.sum(-1, keepdim=True)
    chosen = torch.sort(s + correction, dim=-1, descending=True, stable=True).indices[:, :top]
    picked = torch.gather(s, 1, chosen)
    return chosen, picked / (picked.sum(-1, keepdim=True) + 1e-20)


def experts(h, get, r):
    """The chosen experts' results; the last ``identity`` outputs of the router stand for the input itself."""
    chosen, weight = route(h, get("router"), get("correction"), r["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(r["top"]):
            e = int(chosen[t, j])
            y = h[t] if e >= r["experts"] else gated_unit(h[t][None], get(f"e{e}.gate"), get(f"e{e}.up"), get(f"e{e}.down"))[0]
            out[t] += weight[t, j] * y
    return out


def shared_expert(h, get):
    y = gated_unit(h, get("shared.gate"), get("shared.up"), get("shared.down"))
    return y * sigmoid(h @ get("shared.sg").T)


def moe(h, get, mlp):
    return experts(h, get, mlp["router"]) + shared_expert(h, get)


MIXERS = {"attention": windowed_attention, "latent_attention": latent_attention, "mlstm": lambda *a: mlstm(*a)[0]}


def forward(cfg, tensors, tokens, keep_layers=False):
    """Logits ``[tokens, vocab]`` of one sequence (and the sum of the streams after every layer)."""
    p = {k: v.to(F64) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = p["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    x = x[:, None, :].repeat(1, cfg["streams"], 1)
    stream = []
    for i, layer in enumerate(cfg["layers"]):
        def sublayer(x, which, fn):
            hc = {n: p[f"l{i}.hc{which}.{n}"] for n in ("in", "out", "mix")}
            h = norm_around_zero(gather_streams(x, hc["in"]), p[f"l{i}.norm{which}"], eps)
            return mix_streams(x, fn(h), hc["out"], hc["mix"])
        x = sublayer(x, 1, lambda h: MIXERS[layer["type"]](h, lambda name: p[f"l{i}.mix.{name}"], layer["mixer"], eps))
        if layer.get("mlp") is not None:
            x = sublayer(x, 2, lambda h: moe(h, lambda name: p[f"l{i}.mlp.{name}"], layer["mlp"]))
        stream.append(x.sum(1))
    logits = norm_around_zero(x.sum(1), p["final.norm"], eps) @ p["head"].T * cfg["logit_scale"]
    return (logits, torch.stack(stream)) if keep_layers else logits
