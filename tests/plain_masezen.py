"""A plain, slow Masezen in double precision: one function per mechanism, loops where a loop is the definition.

It works on a nested configuration dictionary and a flat ``{tensor name: tensor}`` dictionary, one unpadded sequence at a
time, and imports nothing from the package: the tests compare the package against it. ``h`` is ``[tokens, width]``.
"""
import math

import torch

F64 = torch.float64


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z * z * z)))


def rms(x, eps):
    """Rows divided by their root mean square, eps under the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def convolve(h, w, before=None):
    """A causal convolution per channel, ``w [width, taps]`` with the current token's tap last; ``before [taps - 1, width]``: the rows
    ahead of the first one (zeros at a sequence's start)."""
    n, taps = h.shape[0], w.shape[1]
    rows = torch.cat([torch.zeros(taps - 1, h.shape[1], dtype=h.dtype) if before is None else before, h])
    out = torch.zeros_like(h)
    for t in range(n):
        for j in range(taps):
            out[t] += w[:, j] * rows[t + j]
    return out


# ------------------------------------------------------------------------------------------ rotation
def frequencies(rot):
    """Angles per position of the rotated pairs, and the factor on sine and cosine."""
    dims, base, y = rot["dims"], rot["base"], rot.get("scaling")
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if y is None:
        return plain, 1.0

    def turning_dim(turns):
        return dims * math.log(y["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(turning_dim(y["fast"])), 0)
    hi = min(math.ceil(turning_dim(y["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / y["factor"] * r + f * (1.0 - r))
    return out, 0.1 * math.log(y["factor"]) + 1.0


def rotate(x, rot, first=0):
    """``x [tokens, heads, dim]``, the first token at position ``first``: dimension ``i`` turns with dimension ``i + dims / 2``."""
    f, size = frequencies(rot)
    half, out = rot["dims"] // 2, x.clone()
    for t in range(x.shape[0]):
        for i in range(half):
            c, s = size * math.cos((first + t) * f[i]), size * math.sin((first + t) * f[i])
            u, v = x[t, :, i], x[t, :, i + half]
            out[t, :, i] = u * c - v * s
            out[t, :, i + half] = v * c + u * s
    return out


# ------------------------------------------------------------------------------------------ attention
def mixed_attention(q, k, v, scale, talk):
    """``q [n, H, dim]`` are the last ``n`` positions of ``k [t, G, dim]`` / ``v [t, G, vdim]``; query head ``h`` reads group
    ``h // (H / G)``. Before the softmax the heads' scores are mixed by ``talk [H, H]``."""
    n, heads, _ = q.shape
    t, groups, vdim = v.shape
    per = heads // groups
    out = torch.zeros(n, heads, vdim, dtype=q.dtype)
    for i in range(n):
        end = t - n + i + 1
        own = torch.stack([k[:end, a // per] @ q[i, a] * scale for a in range(heads)])
        for a in range(heads):
            s = sum(talk[a, g] * own[g] for g in range(heads))
            e = torch.exp(s - s.max())
            out[i, a] = (e @ v[:end, a // per]) / e.sum()
    return out


def attention(h, get, m, eps):
    n, heads, groups, dim = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (h @ get("q").T).reshape(n, heads, dim)
    k = (h @ get("k").T).reshape(n, groups, dim)
    v = k
    q, k = (rotate(rms(t, eps) * get(w), m["rot"]) for t, w in ((q, "q.norm"), (k, "k.norm")))
    o = mixed_attention(q, k, v, m["scale"], get("talk")).reshape(n, -1)
    return (o * sigmoid(h @ get("g").T)) @ get("o").T


# ------------------------------------------------------------------------------------------ feed-forward
def squared_relu_mlp(h, up, down):
    a = torch.clamp(h @ up.T, min=0.0)
    return (a * a) @ down.T


def clamped_expert(h, gate, up, down, limit):
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def route(h, w, top):
    """Per token the chosen experts and their scores."""
    s = sigmoid(h @ w.T)
    chosen = torch.sort(s, dim=-1, descending=True, stable=True).indices[:, :top]
    return chosen, torch.gather(s, 1, chosen)


def moe(h, get, mlp):
    chosen, weight = route(h, get("router"), mlp["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(mlp["router"]["top"]):
            e = int(chosen[t, j])
            out[t] += clamped_expert((weight[t, j] * h[t])[None], get(f"e{e}.gate"), get(f"e{e}.up"), get(f"e{e}.down"),
                                     mlp["expert"]["limit"])[0]
    if mlp.get("shared"):
        out = out + clamped_expert(h, get("shared.gate"), get("shared.up"), get("shared.down"), mlp["shared"]["limit"])
    return out


def feed_forward(h, get, mlp):
    return squared_relu_mlp(h, get("up"), get("down")) if mlp["kind"] == "dense" else moe(h, get, mlp)


# ------------------------------------------------------------------------------------------ a layer
def token_input(x, e, gate, proj, w, eps):
    """What a layer adds to the stream ``x`` from the token's own vector ``e [tokens, dim]``."""
    return rms((gelu_tanh(x @ gate.T) * e) @ proj.T, eps) * w


def layer(x, e, get, spec, eps):
    h = rms(x, eps) * get("norm1")
    out = get("ls1") * attention(h + convolve(h, get("canon1")), lambda n: get("mix." + n), spec["mixer"], eps)
    if spec.get("mlp") is not None:
        out = out + get("ls2") * feed_forward(h, lambda n: get("mlp." + n), spec["mlp"])
    x = x + out
    return x + token_input(x, e, get("side.gate"), get("side.proj"), get("side.norm"), eps)


def forward(cfg, tensors, tokens, keep_layers=False):
    """Logits ``[tokens, vocab]`` of one sequence (and the residual stream after every layer)."""
    p = {k: v.to(F64) for k, v in tensors.items()}
    eps, dim, tokens = cfg["norm"]["eps"], cfg["token_side"]["dim"], torch.as_tensor(tokens)
    x, side, stream = p["embed"][tokens], p["side.embed"][tokens], []
    for i, spec in enumerate(cfg["layers"]):
        x = layer(x, side[:, i * dim:(i + 1) * dim], lambda n: p[f"l{i}.{n}"], spec, eps)
        stream.append(x)
    logits = (rms(x, eps) * p["final.norm"]) @ p["head"].T
    return (logits, torch.stack(stream)) if keep_layers else logits
