"""Small Moronex configurations and random weights for the tests (no two of the sizes of a layer agree unless the case is about that)."""
import json
import os

import torch


def hgrn2(heads, dim, vdim, mlp):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}, "mlp": mlp}


def latent(heads, dim, vdim, q_rank, kv_rank, scale, mlp, kv_from=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def case(vocab, width, eps, *layers):
    return {"architecture": "Moronex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": list(layers)}


CASES = {
    # every branch once; sizes that are multiples of 8
    "mixed": case(96, 48, 1e-5, latent(3, 16, 24, 40, 32, 0.3, moe(24, 5, 2)), hgrn2(2, 24, 16, dense(56)),
                  latent(2, 24, 16, 32, 32, 0.2, dense(40), kv_from=0), hgrn2(3, 16, 8, None)),
    # sizes that are multiples of nothing
    "odd": case(51, 35, 1e-3, hgrn2(3, 7, 5, moe(9, 3, 3)), latent(5, 9, 11, 13, 10, 0.5, dense(17)),
                latent(1, 6, 3, 7, 10, 0.9, moe(11, 4, 1), kv_from=1), latent(2, 4, 13, 9, 15, 0.4, None)),
    # head sizes the tensor-core kernels take as they are
    "heads64": case(128, 128, 1e-5, hgrn2(2, 64, 64, dense(192)), latent(2, 64, 64, 96, 64, 0.125, moe(64, 4, 2)),
                    latent(4, 64, 64, 64, 64, 0.15, dense(128), kv_from=1)),
    # one head, one expert, sizes of 1; two latent layers that are both shared
    "ones": case(17, 16, 1e-6, latent(1, 8, 8, 8, 8, 1.0, moe(8, 1, 1)), latent(1, 8, 8, 8, 8, 1.0, None, kv_from=0),
                 latent(2, 4, 4, 8, 16, 0.5, dense(8)), hgrn2(1, 1, 1, None), latent(2, 4, 4, 8, 16, 0.5, None, kv_from=2)),
}


def shapes(cfg):
    """``{tensor name: shape}`` of a checkpoint of ``cfg``."""
    w, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"]), "head": (cfg["vocab"], cfg["width"]), "final.norm": (cfg["width"],)}
    for i, layer in enumerate(cfg["layers"]):
        m, mlp = layer["mixer"], layer["mlp"]
        h, d, v = m["heads"], m["dim"], m["vdim"]
        mix = {"o": (w, h * v)}
        if layer["type"] == "hgrn2":
            mix.update({"q": (h * d, w), "f": (h * d, w), "f.b": (h * d,), "lower": (h * d,), "v": (h * v, w), "norm": (v,)})
        else:
            mix.update({"dq": (m["q_rank"], w), "dq.norm": (m["q_rank"],), "uq": (h * d, m["q_rank"]), "uk": (h * d, m["kv_rank"]),
                        "uv": (h * v, m["kv_rank"]), "sink": (h,), "g": (h, w)})
            if "kv_from" not in m:
                mix.update({"dkv": (m["kv_rank"], w), "dkv.norm": (m["kv_rank"],)})
        out.update({f"l{i}.mix.{k}": s for k, s in mix.items()})
        for n in ("1", "2") if mlp is not None else ("1",):
            out.update({f"l{i}.norm{n}": (w,), f"l{i}.norm{n}b": (w,), f"l{i}.rg{n}": (w, w), f"l{i}.rg{n}.b": (w,)})
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            ff = {"gate": (mlp["ff"], w), "up": (mlp["ff"], w), "down": (w, mlp["ff"])}
        else:
            e, f = mlp["router"]["experts"], mlp["expert"]["ff"]
            ff = {"router": (e, w), "router.b": (e,)}
            for j in range(e):
                ff.update({f"e{j}.up": (f, w), f"e{j}.down": (w, f)})
        out.update({f"l{i}.mlp.{k}": s for k, s in ff.items()})
    return out


def make_tensors(cfg, seed=0):
    """bfloat16 weights under which every term of the design is visible in the logits."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, s in shapes(cfg).items():
        t = torch.randn(*s, generator=g)
        if name.endswith("lower"):
            t = torch.rand(*s, generator=g) * 0.95
        elif name.endswith("f.b"):
            t = t + 2.0                               # forget slowly
        elif name.endswith("sink"):
            t = t * 1.5
        elif name.endswith(("dq.norm", "dkv.norm", "mix.norm")):
            t = 1.0 + 0.2 * t
        elif name.endswith((".norm1", ".norm2", ".norm1b", ".norm2b", "final.norm")):
            t = 0.2 * t
        elif len(s) == 2 and name != "embed":
            t = t * s[1] ** -0.5 * (1.5 if name.endswith(("uq", "uk")) else 1.0)
        out[name] = t.to(torch.bfloat16)
    return out


def far_key_weights(cfg, layer, tensors):
    """Turn ``layer``'s attention into a search: queries and keys much larger, no help from the sink, so that single far keys
    decide what a position gets."""
    out = dict(tensors)
    out[f"l{layer}.mix.uq"] = out[f"l{layer}.mix.uq"] * 4.0
    out[f"l{layer}.mix.sink"] = out[f"l{layer}.mix.sink"] * 0.0 - 2.0
    return out


def write_model(directory, cfg, tensors):
    from safetensors.torch import save_file
    os.makedirs(directory, exist_ok=True)
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in tensors.items()}, os.path.join(directory, "model.safetensors"))
