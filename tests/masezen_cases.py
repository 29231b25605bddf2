"""Small Masezen configurations and random weights for the tests (no two of the sizes of a layer agree unless the case is about that)."""
import json
import os

import torch

YARN = {"factor": 3.0, "original": 40, "fast": 8.0, "slow": 0.5}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, limit, shared=None, shared_limit=1.5):
    out = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    return out if shared is None else {**out, "shared": {"ff": shared, "limit": shared_limit}}


def attn(heads, kv_heads, dim, scale, rot_dims, mlp, base=10000.0, scaling=None):
    rot = {"dims": rot_dims, "base": base}
    if scaling is not None:
        rot["scaling"] = scaling
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "rot": rot}, "mlp": mlp}


def case(vocab, width, eps, taps, side, *layers):
    return {"architecture": "Masezen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "canon": {"taps": taps},
            "token_side": {"dim": side}, "layers": list(layers)}


CASES = {
    # every branch once; sizes that are multiples of 8
    "mixed": case(96, 48, 1e-5, 3, 16, attn(6, 2, 16, 0.3, 8, dense(56), 500.0, YARN), attn(4, 1, 24, 0.25, 24, moe(24, 5, 2, 1.2, 40, 0.8), 1e4),
                  attn(2, 2, 8, 0.4, 4, None, 100.0, {**YARN, "factor": 8.0}), attn(3, 3, 16, 0.2, 16, moe(16, 6, 3, 2.0), 5e5, YARN)),
    # sizes that are multiples of nothing
    "odd": case(51, 35, 1e-3, 5, 9, attn(5, 5, 7, 0.4, 4, moe(13, 3, 3, 0.9, 17, 2.1), 50.0, {**YARN, "fast": 30.0}), attn(6, 3, 9, 0.3, 6, dense(21)),
                attn(6, 2, 5, 0.5, 2, moe(7, 7, 5, 3.0, 11, 0.5), 300.0), attn(1, 1, 11, 0.3, 10, None, 20.0, YARN)),
    # head sizes the tensor-core kernels take as they are, keys of several widths
    "heads64": case(128, 128, 2e-6, 3, 40, attn(6, 3, 64, 0.15, 48, moe(80, 10, 2, 1.5, 88, 1.0), 3e5, {"factor": 6.0, "original": 48, "fast": 16.0, "slow": 2.0}),
                    attn(8, 4, 32, 0.2, 16, dense(160)), attn(4, 1, 128, 0.1, 96, moe(96, 8, 2, 2.5, 64), 1e5, YARN), attn(6, 6, 16, 0.3, 16, None)),
    # one head, one expert, one tap, sizes of 1; nothing rotated, factor 1
    "ones": case(17, 16, 1e-6, 1, 1, attn(1, 1, 8, 1.0, 0, moe(8, 1, 1, 1.0, 1, 1.0)), attn(2, 1, 2, 1.0, 2, dense(1), 10.0, {**YARN, "factor": 1.0}),
                 attn(2, 2, 1, 1.0, 0, moe(1, 2, 2, 1.0)), attn(1, 1, 2, 0.5, 2, None)),
}


def shapes(cfg):
    """``{tensor name: shape}`` of a checkpoint of ``cfg``."""
    w, side, n = cfg["width"], cfg["token_side"]["dim"], len(cfg["layers"])
    out = {"embed": (cfg["vocab"], w), "side.embed": (cfg["vocab"], n * side), "head": (cfg["vocab"], w), "final.norm": ()}
    unit = lambda ff: {"gate": (ff, w), "up": (ff, w), "down": (w, ff)}                         # noqa: E731
    for i, layer in enumerate(cfg["layers"]):
        m, mlp = layer["mixer"], layer["mlp"]
        values, keys = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
        out.update({f"l{i}.norm1": (), f"l{i}.ls1": (w,), f"l{i}.canon1": (w, cfg["canon"]["taps"]), f"l{i}.side.gate": (side, w),
                    f"l{i}.side.proj": (w, side), f"l{i}.side.norm": (w,)})
        mix = {"q": (values, w), "k": (keys, w), "q.norm": (m["dim"],), "k.norm": (m["dim"],), "talk": (m["heads"], m["heads"]), "g": (values, w), "o": (w, values)}
        out.update({f"l{i}.mix.{k}": s for k, s in mix.items()})
        if mlp is None:
            continue
        out[f"l{i}.ls2"] = (w,)
        if mlp["kind"] == "dense":
            out.update({f"l{i}.mlp.up": (mlp["ff"], w), f"l{i}.mlp.down": (w, mlp["ff"])})
            continue
        out[f"l{i}.mlp.router"] = (mlp["router"]["experts"], w)
        for e in range(mlp["router"]["experts"]):
            out.update({f"l{i}.mlp.e{e}.{k}": s for k, s in unit(mlp["expert"]["ff"]).items()})
        if "shared" in mlp:
            out.update({f"l{i}.mlp.shared.{k}": s for k, s in unit(mlp["shared"]["ff"]).items()})
    return out


def make_tensors(cfg, seed=0):
    """bfloat16 weights under which every term of the design is visible in the logits."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, s in shapes(cfg).items():
        t = torch.randn(s, generator=g)
        end = name.split(".", 1)[-1]
        if end.endswith("talk"):
            t = 0.7 * torch.eye(s[0]) + 0.5 * t / s[0] ** 0.5
        elif end.endswith("norm") or end in ("norm1", "ls1", "ls2"):
            t = 1.0 + 0.25 * t
        elif end == "canon1":
            t = 0.4 * t
        elif len(s) == 2 and name not in ("embed", "side.embed"):
            t = t * s[1] ** -0.5 * (1.5 if end == "mlp.router" or ".e" in end or "shared" in end else 1.0)
        out[name] = t.to(torch.bfloat16)
    return out


def write_model(directory, cfg, tensors):
    from safetensors.torch import save_file
    os.makedirs(directory, exist_ok=True)
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in tensors.items()}, os.path.join(directory, "model.safetensors"))


def steady(tensors):
    """The same model without a router's close calls, for comparisons in 16-bit: logits far apart."""
    return {n: (4.0 * t if n.endswith("mlp.router") else (0.7 * t if ".mlp.e" in n or ".mlp.shared." in n else t)) for n, t in tensors.items()}
