"""Begovik: a decoder whose layers are listed one by one in the configuration.

A layer is a mixer - ``parallel`` (grouped-query attention and linear attention with constant decays side by side), ``wkv``
(recurrence with a bonus) or ``mamba1`` (selective scan) - and a clamped gated feed-forward (or none). Both read the same
residual stream through norms of their own and are added to it together:

    x <- x + m * (mixer(norm1(x)) + ff(norm2(x)))

with ``x`` in fp32 whatever the parameter dtype. The norms of one row differ in their weights only, so the step that adds a
layer's results to the stream also writes both inputs of the next layer (``ops.branch_join``), across block borders.

Checkpoints use flat names (``l3.mix.left.q``, ``l3.mlp.up``, ...); ``convert_checkpoint`` packs them into the modules.
"""
from __future__ import annotations

import copy
from typing import Any, Dict, List, Optional, Sequence

import torch
import torch.nn as nn
from torch import Tensor
from torch.utils.checkpoint import checkpoint

from ... import ops
from ...modeling_utils import PretrainedConfig, PreTrainedModel
from ...ops.reference import Branch
from ...parallel.layers import Embedding, Linear, RMSNorm
from ...parallel.mpu import Layer, LayerPolicy
from ..common import CausalLMHeadMixin, DecoderBackbone, SequenceClassificationMixin, StaticKVCache
from ..mixers import BonusRecurrence, GatedMLP, SelectiveScan, SideBySide

_MIXER_KEYS = {
    "parallel.left": ("heads", "kv_heads", "dim", "vdim", "scale"),
    "parallel.right": ("heads", "dim", "vdim", "decay"),
    "wkv": ("heads", "dim"),
    "mamba1": ("inner", "state", "dt_rank", "conv"),
}


class BegovikConfig(PretrainedConfig):
    """``layers``: one dictionary per layer with ``type`` (``parallel`` | ``wkv`` | ``mamba1``), the mixer's sizes ``mixer`` and the
    feed-forward ``mlp`` (``{"kind": "dense", "ff": ..., "limit": ...}`` or ``None``); ``embedding``: ``{"scale": ...}``; ``norm``:
    ``{"eps": ...}``; ``residual_mult``. A ``wkv`` mixer's ``decay_rank`` may be left to the checkpoint's shapes."""

    model_type = "begovik"
    attribute_map = {"vocab_size": "vocab", "hidden_size": "width", "n_embd": "width"}

    def __init__(self, layers: Optional[List[Dict[str, Any]]] = None, norm: Optional[Dict[str, Any]] = None,
                 embedding: Optional[Dict[str, Any]] = None, residual_mult: float = 1.0, vocab: int = 32000, width: int = 1024,
                 initializer_range: float = 0.02, use_cache: bool = True, tie_word_embeddings: bool = False, **kwargs: Any) -> None:
        self.layers = copy.deepcopy(list(layers or []))         # a checkpoint may add what it alone fixes
        self.norm = dict(norm or {"eps": 1e-5})
        self.embedding = dict(embedding or {"scale": 1.0})
        self.residual_mult = float(residual_mult)
        self.vocab, self.width = vocab, width
        self.initializer_range = initializer_range
        super().__init__(use_cache=use_cache, tie_word_embeddings=tie_word_embeddings, **kwargs)
        self.check()

    @property
    def eps(self) -> float:
        return float(self.norm["eps"])

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def check(self) -> None:
        """Reject what no layer of the model implements, by layer."""
        for i, layer in enumerate(self.layers):
            kind, m, mlp = layer.get("type"), layer.get("mixer") or {}, layer.get("mlp")
            if kind not in ("parallel", "wkv", "mamba1"):
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            halves = [(f"{kind}.{s}", m.get(s) or {}) for s in ("left", "right")] if kind == "parallel" else [(kind, m)]
            for name, part in halves:
                missing = [k for k in _MIXER_KEYS[name] if k not in part]
                if missing:
                    raise ValueError(f"layer {i}: {name} without {missing}")
            if kind == "parallel":
                left, right, rot = m["left"], m["right"], m["left"].get("rot")
                if left["heads"] % left["kv_heads"]:
                    raise ValueError(f"layer {i}: {left['heads']} query heads over {left['kv_heads']} key / value heads")
                if rot is not None and (rot["dims"] % 2 or not 0 <= rot["dims"] <= left["dim"]):
                    raise ValueError(f"layer {i}: {rot['dims']} rotated of {left['dim']} dims")
                if len(right["decay"]) != right["heads"]:
                    raise ValueError(f"layer {i}: {len(right['decay'])} decays for {right['heads']} heads")
            if mlp is not None and mlp.get("kind") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            if mlp is not None and ("ff" not in mlp or "limit" not in mlp):
                raise ValueError(f"layer {i}: feed-forward without ff or limit")


def _mixer(kind: str, m: Dict[str, Any], width: int, eps: float) -> nn.Module:
    if kind == "wkv":
        return BonusRecurrence(width, m["heads"], m["dim"], eps, **({"decay_rank": m["decay_rank"]} if "decay_rank" in m else {}))
    if kind == "mamba1":
        return SelectiveScan(width, m["inner"], m["state"], m["dt_rank"], m["conv"])
    left = {k: m["left"][k] for k in _MIXER_KEYS["parallel.left"]}
    rot = m["left"].get("rot")
    if rot is not None:
        left.update(rot_dims=rot["dims"], rot_base=rot["base"])
    left["softcap"] = m["left"].get("softcap") or 0.0
    return SideBySide(width, left, {k: m["right"][k] for k in _MIXER_KEYS["parallel.right"]}, eps)


class BegovikBlock(nn.Module):
    oslo_fused = False

    def __init__(self, config: BegovikConfig, layer_id: int) -> None:
        super().__init__()
        spec, w, eps = config.layers[layer_id], config.width, config.eps
        mlp = spec.get("mlp")
        self.kind, self.eps, self.layer_id, self.mult = spec["type"], eps, layer_id, config.residual_mult
        self.norm1 = RMSNorm(w, eps)
        self.mixer = _mixer(self.kind, spec["mixer"], w, eps)
        self.norm2 = RMSNorm(w, eps) if mlp is not None else None
        self.mlp = GatedMLP(w, mlp["ff"], limit=mlp["limit"]) if mlp is not None else None

    def norms(self) -> List[RMSNorm]:
        """What this block wants of the residual stream."""
        return [self.norm1] if self.norm2 is None else [self.norm1, self.norm2]

    def forward(self, x: Tensor, normed: Optional[Sequence[Tensor]] = None, next_norms: Sequence[RMSNorm] = (),
                cache: Optional[StaticKVCache] = None, keep: Optional[Tensor] = None, positions: Optional[Tensor] = None,
                output_attentions: bool = False):
        """``x`` ``[batch, S, width]`` fp32. ``normed``: ``x`` through this block's ``norms()`` when the previous block computed that;
        ``next_norms``: the norms that follow this block. Returns ``(x, [x through next_norms], attention weights or None)``."""
        batch, s, w = x.shape
        rows = x.reshape(batch * s, w)
        if normed is None:
            normed = [n(rows) for n in self.norms()]
        normed = [h.reshape(batch * s, w) for h in normed]
        if self.kind == "parallel":
            out = self.mixer(normed[0], batch, self.layer_id, cache, keep, positions, output_attentions)
        else:
            out = self.mixer(normed[0], batch, self.layer_id, cache, keep)
        branches = list(out.branches) if out.y is None else [Branch(out.y)]
        if self.mlp is not None:
            branches.append(Branch(self.mlp(normed[1]).y))
        rows, after = ops.branch_join(rows, branches, self.mult, self.eps, [n.weight for n in next_norms], fused=self.oslo_fused)
        return rows.view(batch, s, w), [h.view(batch, s, w) for h in after], out.probs


class BegovikPreTrainedModel(PreTrainedModel):
    config_class = BegovikConfig
    base_model_prefix = "transformer"

    def get_layer_policies(self):
        return [BegovikLayerPolicy]

    def _exec_both_engines(self, tensor_parallel_size: int = 1, pipeline_parallel_size: int = 1, **kw: Any):
        if int(tensor_parallel_size) > 1 or int(pipeline_parallel_size) > 1:
            raise NotImplementedError("Begovik runs on one GPU per replica: its packed projections and recurrent states have no "
                                      "tensor- or pipeline-parallel layout (data parallelism works)")
        return super()._exec_both_engines(tensor_parallel_size=1, pipeline_parallel_size=1, **kw)

    def convert_checkpoint(self, state_dict: Dict[str, Tensor]) -> Dict[str, Tensor]:
        """Flat checkpoint names -> module names. Every tensor must be there, with its shape, and none may be left over."""
        if "embed" not in state_dict:
            self._adopt_decay_ranks(lambda i: state_dict.get(f"transformer.h.{i}.mixer.w1.weight", state_dict.get(f"h.{i}.mixer.w1.weight")))
            return state_dict                              # saved by this package
        src = dict(state_dict)
        model = self.base_model
        out: Dict[str, Tensor] = {}

        def take(name: str, shape=None) -> Tensor:
            if name not in src:
                raise KeyError(f"checkpoint has no tensor {name!r}")
            t = src.pop(name)
            if shape is not None and tuple(t.shape) != tuple(shape):
                raise ValueError(f"{name}: shape {tuple(t.shape)}, expected {tuple(shape)}")
            return t

        def put(name: str, param: Tensor, source: str) -> None:
            out[f"transformer.{name}"] = take(source, param.shape)

        self._adopt_decay_ranks(lambda i: src.get(f"l{i}.mix.w1"))
        put("wte.weight", model.wte.weight, "embed")
        put("ln_f.weight", model.ln_f.weight, "final.norm")
        for i, b in enumerate(model.h):
            at, mx, mixer = f"h.{i}.", f"l{i}.mix.", b.mixer
            mat = at + "mixer."
            put(f"{at}norm1.weight", b.norm1.weight, f"l{i}.norm1")
            if b.kind == "parallel":
                parts = {n: take(mx + n) for n in mixer.in_proj.parts}
                out[f"transformer.{mat}in_proj.weight"] = mixer.in_proj.pack(parts)
                for n in ("q", "k"):
                    put(f"{mat}left.{n}_norm.weight", getattr(mixer.left, f"{n}_norm").weight, f"{mx}left.{n}.norm")
                put(f"{mat}right.o_norm.weight", mixer.right.o_norm.weight, mx + "right.norm")
                for side in ("left", "right"):
                    put(f"{mat}{side}.out_proj.weight", getattr(mixer, side).out_proj.weight, f"{mx}{side}.o")
                    put(f"{mat}{side}_norm.weight", getattr(mixer, f"{side}_norm").weight, f"{mx}{side}.out")
            else:
                put(f"{mat}out_proj.weight", mixer.out_proj.weight, mx + "o")
            if b.kind == "wkv":
                width, n = mixer.mu.size(1), mixer.heads * mixer.dim
                out[f"transformer.{mat}mu"] = torch.stack([take(f"{mx}mu.{s}", (width,)) for s in mixer.MIXES])
                out[f"transformer.{mat}rkvg.weight"] = torch.stack([take(mx + s, (n, width)) for s in mixer.MIXES[:4]])
                for name, source in (("w1.weight", "w1"), ("w2.weight", "w2"), ("w0", "w0"), ("o_norm", "norm")):
                    put(mat + name, mixer.get_parameter(name), mx + source)
                out[f"transformer.{mat}u"] = take(mx + "u", (mixer.heads, mixer.dim)).reshape(-1)
            elif b.kind == "mamba1":
                for packed, source in ((mixer.in_proj, "in"), (mixer.x_proj, "x")):
                    sizes = [size for _, size in packed.parts.values()]
                    whole = take(mx + source, (sum(sizes), packed.in_features))
                    name = "in_proj" if packed is mixer.in_proj else "x_proj"
                    out[f"transformer.{mat}{name}.weight"] = packed.pack(dict(zip(packed.parts, whole.split(sizes))))
                for name, source in (("conv_weight", "conv"), ("conv_bias", "conv.b"), ("dt_proj.weight", "dt"), ("dt_bias", "dt.b"),
                                     ("a_log", "A_log"), ("d", "D")):
                    put(mat + name, mixer.get_parameter(name), mx + source)
            if b.mlp is not None:
                put(f"{at}norm2.weight", b.norm2.weight, f"l{i}.norm2")
                parts = {n: take(f"l{i}.mlp.{n}") for n in b.mlp.in_proj.parts}
                out[f"transformer.{at}mlp.in_proj.weight"] = b.mlp.in_proj.pack(parts)
                put(f"{at}mlp.down.weight", b.mlp.down.weight, f"l{i}.mlp.down")
        head = src.pop("head", None)
        if isinstance(self, BegovikForCausalLM):
            if head is None:
                raise KeyError("checkpoint has no tensor 'head'")
            out["lm_head.weight"] = head
        if src:
            raise KeyError(f"checkpoint tensors that no layer of the configuration uses: {sorted(src)[:8]}")
        return out

    def _adopt_decay_ranks(self, w1) -> None:
        """The decay projections' rank is a matter of the checkpoint: ``w1(layer)`` is that layer's first projection or ``None``."""
        for i, b in enumerate(self.base_model.h):
            if b.kind == "wkv" and w1(i) is not None:
                b.mixer.set_decay_rank(w1(i).shape[0])
                self.config.layers[i]["mixer"]["decay_rank"] = int(w1(i).shape[0])


class BegovikModel(DecoderBackbone, BegovikPreTrainedModel):
    def __init__(self, config: BegovikConfig) -> None:
        super().__init__(config)
        self.wte = Embedding(config.vocab, config.width)
        self.h = nn.ModuleList([BegovikBlock(config, i) for i in range(len(config.layers))])
        self.ln_f = RMSNorm(config.width, config.eps)
        self.post_init()

    def embed(self, input_ids, position_ids, token_type_ids, inputs_embeds):
        hs = self.wte(input_ids) if inputs_embeds is None else inputs_embeds
        return hs.to(torch.float32) * float(self.config.embedding["scale"])      # the residual stream is fp32

    def prepare_fn(self, past_key_values=None, use_cache=None, token_type_ids=None, head_mask=None, **kw):
        if token_type_ids is not None or head_mask is not None:
            raise ValueError("Begovik has neither token types nor head masks")
        use_cache = self.config.use_cache if use_cache is None else use_cache
        if past_key_values is not None and not isinstance(past_key_values, StaticKVCache):
            raise TypeError("Begovik continues from a StaticKVCache (what its outputs return)")
        if past_key_values is None and use_cache and not (self.training and torch.is_grad_enabled()):
            ref = next((kw[k] for k in ("input_ids", "inputs_embeds", "hidden_states") if kw.get(k) is not None), None)
            past_key_values = StaticKVCache(ref.shape[1] if ref is not None and ref.dim() > 1 else 1, grow=True)
        kw = super().prepare_fn(past_key_values=past_key_values, use_cache=use_cache, **kw)
        kw["presents"] = None
        kw["_normed"] = None
        if kw["attention_mask"] is not None:
            kw["attention_mask"] = (kw["attention_mask"] != 0).to(torch.uint8)
        return kw

    def block_fn(self, layer_id: int, **kw) -> Dict[str, Any]:
        block = self.h[layer_id]
        hs = kw["hidden_states"]
        if kw["all_hidden_states"] is not None:
            kw["all_hidden_states"].append(hs)
        last = layer_id + 1 == len(self.h)
        args = dict(next_norms=[self.ln_f] if last else self.h[layer_id + 1].norms(), cache=kw["cache"], keep=kw["attention_mask"],
                    positions=kw["position_ids"], output_attentions=kw["output_attentions"])
        if self.gradient_checkpointing and self.training and torch.is_grad_enabled():
            hs, normed, probs = checkpoint(lambda x, n: block(x, n, **args), hs, kw["_normed"], use_reentrant=False)
        else:
            hs, normed, probs = block(hs, kw["_normed"], **args)
        kw["hidden_states"], kw["_normed"] = hs, normed
        if kw["all_attentions"] is not None:
            kw["all_attentions"].append(probs)
        return kw

    def postblock_fn(self, **kw) -> Dict[str, Any]:
        hs = kw["_normed"][0] if kw["_normed"] else self.ln_f(kw["hidden_states"])
        if kw["all_hidden_states"] is not None:
            kw["all_hidden_states"].append(kw["hidden_states"])
        if kw["cache"] is not None:
            kw["cache"].advance(kw["_seq"])
        kw["hidden_states"] = hs
        return kw


class BegovikForCausalLM(CausalLMHeadMixin, BegovikPreTrainedModel):
    def __init__(self, config: BegovikConfig) -> None:
        super().__init__(config)
        self.transformer = BegovikModel(config)
        self.lm_head = Linear(config.width, config.vocab, bias=False)
        self.post_init()

    def get_head_layers(self) -> List[Layer]:
        return [Layer(module=self.lm_head, weight=self.lm_head.weight, parallel=False)]


class BegovikForSequenceClassification(SequenceClassificationMixin, BegovikPreTrainedModel):
    def __init__(self, config: BegovikConfig) -> None:
        super().__init__(config)
        self.num_labels = config.num_labels
        self.transformer = BegovikModel(config)
        self.score = Linear(config.width, self.num_labels, bias=False)
        self.post_init()

    def get_head_layers(self) -> List[Layer]:
        return [Layer(module=self.score, weight=self.score.weight, parallel=False)]


class BegovikLayerPolicy(LayerPolicy):
    """Where the layers are (``fuse()`` only flips the building blocks' ``oslo_fused``; there is no tensor-parallel layout)."""

    @staticmethod
    def word_embedding(model, config):
        wte = model.base_model.wte
        return [Layer(module=wte, weight=wte.weight, parallel=False)]

    @staticmethod
    def block_layers(model, config):
        return list(model.base_model.h)

    @staticmethod
    def postblock_layers(model, config):
        ln = model.base_model.ln_f
        return [Layer(module=ln, weight=ln.weight, parallel=False)]

    @staticmethod
    def original_layer_class():
        return BegovikBlock
