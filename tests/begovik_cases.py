"""Small Begovik configurations and random weights for the tests (no two of the sizes of a layer agree unless the case is about that)."""
import json
import os

import torch


def dense(ff, limit=1.5):
    return {"kind": "dense", "ff": ff, "limit": limit}


def wkv(heads, dim, mlp, rank=12):
    """``rank`` of the decay projections: not part of a configuration, only of the weights."""
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": mlp, "_rank": rank}


def mamba(inner, state, dt_rank, conv, mlp):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}, "mlp": mlp}


def attn(heads, kv_heads, dim, vdim, scale, softcap, rot_dims, base=10000.0):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap,
            "rot": {"dims": rot_dims, "base": base}}


def lin(heads, dim, vdim, decay):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}


def parallel(left, right, mlp):
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": mlp}


def case(vocab, width, eps, *layers, scale=3.0, mult=0.4):
    return {"architecture": "Begovik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "residual_mult": mult, "layers": list(layers)}


def public(cfg):
    """The configuration as a checkpoint has it."""
    return {**cfg, "layers": [{k: v for k, v in l.items() if not k.startswith("_")} for l in cfg["layers"]]}


CASES = {
    # every branch once; sizes that are multiples of 8
    "mixed": case(96, 48, 1e-5, parallel(attn(6, 2, 16, 24, 0.3, 8.0, 8), lin(3, 24, 16, (0.5, 0.9, 0.99)), dense(56)),
                  wkv(2, 24, dense(40), 16), mamba(64, 16, 8, 4, dense(72, 0.7)), wkv(4, 16, None, 8), mamba(40, 8, 16, 3, None),
                  parallel(attn(2, 2, 24, 16, 0.2, 20.0, 24, 500.0), lin(2, 16, 40, (0.0, 1.0)), None)),
    # sizes that are multiples of nothing
    "odd": case(51, 35, 1e-3, mamba(27, 5, 3, 2, dense(17, 0.9)), parallel(attn(5, 1, 9, 11, 0.5, 3.0, 6), lin(3, 7, 5, (0.3, 0.8, 0.97)), dense(13)),
                wkv(3, 7, dense(19), 5), mamba(33, 19, 7, 5, dense(11)), parallel(attn(6, 3, 6, 3, 0.9, 30.0, 2), lin(1, 4, 13, (0.95,)), None),
                wkv(1, 21, None, 1), scale=1.7, mult=1.0),
    # head sizes the tensor-core kernels take as they are, groups of several sizes
    "heads64": case(128, 128, 1e-5, parallel(attn(4, 1, 64, 64, 0.125, 15.0, 64), lin(2, 64, 64, (0.7, 0.98)), dense(192)),
                    wkv(2, 64, dense(128), 32), parallel(attn(2, 2, 128, 128, 0.09, 40.0, 32), lin(1, 128, 64, (0.999,)), dense(64)),
                    mamba(256, 16, 16, 4, dense(96)), parallel(attn(8, 2, 64, 32, 0.125, 15.0, 16), lin(4, 32, 32, (0.4, 0.6, 0.8, 0.9)), None)),
    # one head, one channel, one tap, sizes of 1; neither rotation nor cap
    "ones": case(17, 16, 1e-6, parallel({"heads": 1, "kv_heads": 1, "dim": 8, "vdim": 8, "scale": 1.0}, lin(1, 1, 1, (0.5,)), dense(8)),
                 wkv(1, 1, dense(8), 2), mamba(8, 1, 1, 1, dense(1)), wkv(2, 8, None, 16), scale=1.0, mult=1.0),
}


def shapes(cfg):
    """``{tensor name: shape}`` of a checkpoint of ``cfg``."""
    w, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"]), "head": (cfg["vocab"], cfg["width"]), "final.norm": (cfg["width"],)}
    for i, layer in enumerate(cfg["layers"]):
        m, mlp = layer["mixer"], layer["mlp"]
        if layer["type"] == "wkv":
            n = m["heads"] * m["dim"]
            mix = {s: (n, w) for s in "rkvg"}
            mix.update({f"mu.{s}": (w,) for s in "rkvgw"})
            mix.update({"w1": (layer["_rank"], w), "w2": (n, layer["_rank"]), "w0": (n,), "u": (m["heads"], m["dim"]), "norm": (n,), "o": (w, n)})
        elif layer["type"] == "mamba1":
            c, s, r = m["inner"], m["state"], m["dt_rank"]
            mix = {"in": (2 * c, w), "conv": (c, m["conv"]), "conv.b": (c,), "x": (r + 2 * s, c), "dt": (c, r), "dt.b": (c,),
                   "A_log": (c, s), "D": (c,), "o": (w, c)}
        else:
            a, b = m["left"], m["right"]
            mix = {"left.q": (a["heads"] * a["dim"], w), "left.k": (a["kv_heads"] * a["dim"], w), "left.v": (a["kv_heads"] * a["vdim"], w),
                   "left.q.norm": (a["dim"],), "left.k.norm": (a["dim"],), "left.o": (w, a["heads"] * a["vdim"])}
            n = b["heads"] * b["vdim"]
            mix.update({"right.q": (b["heads"] * b["dim"], w), "right.k": (b["heads"] * b["dim"], w), "right.v": (n, w), "right.g": (n, w),
                        "right.norm": (n,), "right.o": (w, n), "left.out": (w,), "right.out": (w,)})
        out.update({f"l{i}.mix.{k}": s for k, s in mix.items()})
        out[f"l{i}.norm1"] = (w,)
        if mlp is not None:
            out[f"l{i}.norm2"] = (w,)
            out.update({f"l{i}.mlp.gate": (mlp["ff"], w), f"l{i}.mlp.up": (mlp["ff"], w), f"l{i}.mlp.down": (w, mlp["ff"])})
    return out


def make_tensors(cfg, seed=0):
    """bfloat16 weights under which every term of the design is visible in the logits."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, s in shapes(cfg).items():
        t = torch.randn(*s, generator=g)
        end = name.split(".", 1)[-1]
        if ".mu." in name:
            t = torch.rand(*s, generator=g)
        elif end == "mix.w0":
            t = 1.5 * t - 3.0                             # decays from hardly any to much
        elif end == "mix.u":
            t = t + 0.5
        elif end == "mix.dt.b":
            t = t - 2.0
        elif end == "mix.A_log":
            t = 0.7 * t + 0.3
        elif end == "mix.D":
            t = 1.0 + 0.5 * t
        elif end == "mix.conv":
            t = t * s[1] ** -0.5
        elif end == "mix.conv.b":
            t = 0.3 * t
        elif end.endswith("norm") or end in ("norm1", "norm2", "mix.left.out", "mix.right.out"):
            t = 1.0 + 0.2 * t
        elif len(s) == 2 and name != "embed":
            t = t * s[1] ** -0.5 * (2.0 if end in ("mlp.gate", "mlp.up", "mix.w2") else 1.0)
        out[name] = t.to(torch.bfloat16)
    return out


def far_key_weights(layer, tensors, factor=4.0):
    """Turn ``layer``'s attention into a search: normed queries and keys much larger, so that single far keys decide what a
    position gets."""
    out = dict(tensors)
    for n in ("q", "k"):
        name = f"l{layer}.mix.left.{n}.norm"
        out[name] = out[name] * factor
    return out


def write_model(directory, cfg, tensors):
    from safetensors.torch import save_file
    os.makedirs(directory, exist_ok=True)
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(public(cfg), f)
    save_file({k: v.contiguous() for k, v in tensors.items()}, os.path.join(directory, "model.safetensors"))
