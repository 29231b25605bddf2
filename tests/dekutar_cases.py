"""Small Dekutar configurations and random weights for the tests (no two of the sizes of a layer agree unless the case is about that)."""
import json
import os

import torch


def moe(ff, experts, identity, top, shared):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top}, "shared": {"ff": shared}}


def attn(heads, kv_heads, dim, scale, size, keep_first, rot_dims, mlp, base=10000.0):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale,
                                           "mask": {"size": size, "keep_first": keep_first}, "rot": {"dims": rot_dims, "base": base}}, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, mlp, base=500.0):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank,
                                                  "kv_rank": kv_rank, "scale": scale, "rot": {"dims": rot_dim, "base": base}}, "mlp": mlp}


def mlstm(heads, dim, vdim, cap, mlp):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


def case(vocab, width, eps, streams, *layers, scale=2.0, logit_scale=0.7):
    return {"architecture": "Dekutar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "streams": streams, "logit_scale": logit_scale, "layers": list(layers)}


CASES = {
    # every branch once; sizes that are multiples of 8
    "mixed": case(96, 48, 1e-5, 3, attn(6, 2, 16, 0.3, 7, 3, 8, moe(24, 5, 2, 3, 40)), mlstm(3, 24, 16, 9.0, moe(16, 6, 1, 2, 56)),
                  latent(3, 16, 8, 24, 40, 32, 0.25, moe(32, 4, 3, 4, 24)), mlstm(2, 8, 40, 15.0, None),
                  latent(4, 8, 24, 16, 24, 48, 0.2, None), attn(2, 2, 24, 0.2, 11, 0, 24, None, 500.0)),
    # sizes that are multiples of nothing
    "odd": case(51, 35, 1e-3, 5, mlstm(3, 7, 5, 4.0, moe(13, 3, 2, 2, 17)), attn(5, 1, 9, 0.5, 6, 2, 6, moe(7, 7, 1, 5, 11)),
                latent(3, 5, 6, 11, 13, 9, 0.4, moe(9, 5, 4, 3, 5)), attn(6, 3, 6, 0.9, 1, 5, 2, moe(11, 2, 1, 1, 3)),
                latent(1, 3, 2, 7, 5, 17, 0.6, None), mlstm(1, 13, 3, 30.0, None), scale=1.7, logit_scale=1.3),
    # head sizes the tensor-core kernels take as they are, groups of several sizes
    "heads64": case(128, 128, 1e-6, 2, latent(4, 64, 64, 128, 96, 64, 0.1, moe(64, 12, 5, 4, 88)), attn(4, 1, 128, 0.1, 33, 9, 64, moe(96, 8, 0, 2, 64)),
                    mlstm(2, 64, 128, 12.0, moe(48, 6, 2, 6, 128)), latent(2, 128, 64, 64, 64, 128, 0.08, moe(32, 4, 4, 2, 32)),
                    attn(8, 4, 64, 0.13, 24, 17, 16, None), mlstm(4, 32, 32, 6.0, None)),
    # one stream, one head, one expert, sizes of 1; windows of one position, nothing kept, no identity experts
    "ones": case(17, 16, 1e-6, 1, attn(1, 1, 8, 1.0, 1, 0, 0, moe(8, 1, 0, 1, 8)), mlstm(1, 1, 1, 1.0, moe(1, 2, 1, 1, 1)),
                 latent(1, 1, 2, 1, 1, 1, 1.0, moe(8, 1, 3, 4, 1)), attn(2, 1, 2, 1.0, 2, 1, 2, None), scale=1.0, logit_scale=1.0),
}


def shapes(cfg):
    """``{tensor name: shape}`` of a checkpoint of ``cfg``."""
    w, n, out = cfg["width"], cfg["streams"], {"embed": (cfg["vocab"], cfg["width"]), "head": (cfg["vocab"], cfg["width"]), "final.norm": (cfg["width"],)}
    for i, layer in enumerate(cfg["layers"]):
        m, mlp, heads = layer["mixer"], layer["mlp"], layer["mixer"]["heads"]
        values = heads * m["vdim"]
        if layer["type"] == "attention":
            mix = {"q": (heads * m["dim"], w), "k": (m["kv_heads"] * m["dim"], w), "g": (heads, w)}
        elif layer["type"] == "latent_attention":
            mix = {"dq": (m["q_rank"], w), "dq.norm": (m["q_rank"],), "uq": (heads * (m["dim"] + m["rot_dim"]), m["q_rank"]),
                   "dkv": (m["kv_rank"] + m["rot_dim"], w), "dkv.norm": (m["kv_rank"],), "uk": (heads * m["dim"], m["kv_rank"]),
                   "uv": (values, m["kv_rank"]), "g": (values, w)}
        else:
            mix = {"q": (heads * m["dim"], w), "k": (heads * m["dim"], w), "v": (values, w), "g": (values, w), "norm": (values,),
                   "i": (heads, w), "i.b": (heads,), "f": (heads, w), "f.b": (heads,)}
        mix["o"] = (w, values)
        out.update({f"l{i}.mix.{k}": s for k, s in mix.items()})
        for q in ("1", "2") if mlp is not None else ("1",):
            out.update({f"l{i}.norm{q}": (w,), f"l{i}.hc{q}.in": (n,), f"l{i}.hc{q}.out": (n,), f"l{i}.hc{q}.mix": (n, n)})
        if mlp is not None:
            unit = lambda ff: {"gate": (ff, w), "up": (ff, w), "down": (w, ff)}                 # noqa: E731
            for e in range(mlp["router"]["experts"]):
                out.update({f"l{i}.mlp.e{e}.{k}": s for k, s in unit(mlp["expert"]["ff"]).items()})
            outputs = mlp["router"]["experts"] + mlp["router"]["identity"]
            out.update({f"l{i}.mlp.router": (outputs, w), f"l{i}.mlp.correction": (outputs,), f"l{i}.mlp.shared.sg": (1, w)})
            out.update({f"l{i}.mlp.shared.{k}": s for k, s in unit(mlp["shared"]["ff"]).items()})
    return out


def make_tensors(cfg, seed=0):
    """bfloat16 weights under which every term of the design is visible in the logits."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, s in shapes(cfg).items():
        t = torch.randn(*s, generator=g)
        end = name.split(".", 1)[-1]
        if end in ("hc1.in", "hc2.in"):
            t = (1.0 + 0.3 * t) / s[0]
        elif end in ("hc1.out", "hc2.out"):
            t = 1.0 + 0.4 * t
        elif end in ("hc1.mix", "hc2.mix"):
            t = 0.8 * torch.eye(s[0]) + 0.2 * t
        elif end == "mix.i.b":
            t = 2.0 * t
        elif end == "mix.f.b":
            t = 2.0 * t + 2.5                             # from forgetting at once to hardly at all
        elif end == "mlp.correction":
            t = 0.2 * t
        elif end in ("norm1", "norm2", "norm"):           # stored around zero
            t = 0.2 * t
        elif end.endswith(".norm"):
            t = 1.0 + 0.2 * t
        elif len(s) == 2 and name != "embed":
            t = t * s[1] ** -0.5 * (2.0 if end in ("mlp.router", "mix.i", "mix.f") or ".e" in end or "shared" in end else 1.0)
        out[name] = t.to(torch.bfloat16)
    return out


def write_model(directory, cfg, tensors):
    from safetensors.torch import save_file
    os.makedirs(directory, exist_ok=True)
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in tensors.items()}, os.path.join(directory, "model.safetensors"))


def steady(tensors):
    """The same model without a router's close calls, for comparisons in 16-bit: corrections far apart choose, scores only weigh."""
    out = dict(tensors)
    for name, t in tensors.items():
        if name.endswith("mlp.correction"):
            g = torch.Generator().manual_seed(t.numel())
            out[name] = (1.5 * torch.randperm(t.numel(), generator=g)).to(t.dtype)
        elif ".mlp.e" in name or ".mlp.shared." in name:
            out[name] = 0.7 * t
    return out
