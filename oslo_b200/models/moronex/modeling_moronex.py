"""Moronex: a decoder whose layers are listed one by one in the configuration.

A layer is a mixer - latent attention without positions (optionally over another layer's latents) or a gated linear
recurrence - and a feed-forward (dense gated, mixture of experts, or none). Both sublayers are normed before and after
and gated by a sigmoid projection of their own input:

    x <- x + norm_post(mixer(h) * sigmoid(W_rg h + b_rg)),   h = norm_pre(x)

with the residual stream ``x`` in fp32 whatever the parameter dtype. The residual-gate projection rides in each
sublayer's packed input GEMM, and gate, post-norm, residual addition and the next sublayer's pre-norm are one kernel
(``ops.residual_join``), across block borders too.

Checkpoints use flat names (``l3.mix.q``, ``l3.mlp.e0.up``, ...); ``convert_checkpoint`` packs them into the modules.
"""
from __future__ import annotations

import re
from typing import Any, Dict, List, Optional

import torch
import torch.nn as nn
from torch import Tensor
from torch.utils.checkpoint import checkpoint

from ... import ops
from ...modeling_utils import PretrainedConfig, PreTrainedModel
from ...parallel.layers import Embedding, Linear, RMSNorm
from ...parallel.mpu import Layer, LayerPolicy
from ..common import CausalLMHeadMixin, DecoderBackbone, SequenceClassificationMixin, StaticKVCache
from ..mixers import GatedLinearRecurrence, GatedMLP, LatentAttention, MixtureOfExperts


class MoronexConfig(PretrainedConfig):
    """``layers``: one dictionary per layer with ``type`` (``latent_attention`` | ``hgrn2``), the mixer's sizes ``mixer`` and the
    feed-forward ``mlp`` (``{"kind": "dense", "ff": ...}``, ``{"kind": "moe", "expert": {"ff": ...}, "router": {"experts": ...,
    "top": ...}}`` or ``None``); ``norm``: ``{"eps": ...}``."""

    model_type = "moronex"
    attribute_map = {"vocab_size": "vocab", "hidden_size": "width", "n_embd": "width"}

    def __init__(self, layers: Optional[List[Dict[str, Any]]] = None, norm: Optional[Dict[str, Any]] = None, vocab: int = 32000,
                 width: int = 1024, initializer_range: float = 0.02, use_cache: bool = True, tie_word_embeddings: bool = False,
                 **kwargs: Any) -> None:
        self.layers = list(layers or [])
        self.norm = dict(norm or {"eps": 1e-5})
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
            need = {"latent_attention": ("heads", "dim", "vdim", "q_rank", "kv_rank", "scale"), "hgrn2": ("heads", "dim", "vdim")}
            if kind not in need:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            missing = [k for k in need[kind] if k not in m]
            if missing:
                raise ValueError(f"layer {i}: mixer without {missing}")
            src = m.get("kv_from")
            if src is not None:
                ok = (kind == "latent_attention" and 0 <= src < i and self.layers[src].get("type") == "latent_attention"
                      and self.layers[src]["mixer"].get("kv_from") is None
                      and self.layers[src]["mixer"]["kv_rank"] == m["kv_rank"])
                if not ok:
                    raise ValueError(f"layer {i}: kv_from {src} is not an earlier latent-attention layer with latents of its own "
                                     "and the same kv_rank")
            if mlp is not None:
                if mlp.get("kind") not in ("dense", "moe"):
                    raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
                if mlp["kind"] == "moe" and not 1 <= mlp["router"]["top"] <= mlp["router"]["experts"]:
                    raise ValueError(f"layer {i}: top {mlp['router']['top']} of {mlp['router']['experts']} experts")


class MoronexBlock(nn.Module):
    oslo_fused = False

    def __init__(self, config: MoronexConfig, layer_id: int) -> None:
        super().__init__()
        spec = config.layers[layer_id]
        m, mlp, w, eps = spec["mixer"], spec.get("mlp"), config.width, config.eps
        self.kind, self.eps, self.layer_id = spec["type"], eps, layer_id
        self.kv_layer = m.get("kv_from") if m.get("kv_from") is not None else layer_id
        side = {"rg": w}                                   # the residual gate reads the sublayer's input
        self.norm1 = RMSNorm(w, eps, offset=1.0)
        self.norm1b = RMSNorm(w, eps, offset=1.0)
        self.rg1_bias = nn.Parameter(torch.zeros(w))
        if self.kind == "latent_attention":
            self.mixer = LatentAttention(w, m["heads"], m["dim"], m["vdim"], m["q_rank"], m["kv_rank"], m["scale"], eps,
                                         shared_latents=self.kv_layer != layer_id, side=side)
        else:
            self.mixer = GatedLinearRecurrence(w, m["heads"], m["dim"], m["vdim"], eps, side=side)
        self.mlp = None
        if mlp is not None:
            self.norm2 = RMSNorm(w, eps, offset=1.0)
            self.norm2b = RMSNorm(w, eps, offset=1.0)
            self.rg2_bias = nn.Parameter(torch.zeros(w))
            if mlp["kind"] == "dense":
                self.mlp = GatedMLP(w, mlp["ff"], side=side)
            else:
                self.mlp = MixtureOfExperts(w, mlp["expert"]["ff"], mlp["router"]["experts"], mlp["router"]["top"], side=side)

    def _join(self, x, y, gate, gate_bias, norm, nxt, slots=None, weights=None):
        fn = ops.residual_join if self.oslo_fused else ops.reference.residual_join
        return fn(x, y, gate, gate_bias, norm.weight, nxt.weight if nxt is not None else None, self.eps, slots, weights)

    def forward(self, x: Tensor, normed: Optional[Tensor] = None, next_norm: Optional[RMSNorm] = None,
                latent: Optional[Tensor] = None, cache: Optional[StaticKVCache] = None, keep: Optional[Tensor] = None,
                output_attentions: bool = False):
        """``x`` ``[batch, S, width]`` fp32. ``normed``: this block's ``norm1`` of ``x`` when the previous block computed it;
        ``next_norm``: the norm that follows this block. Returns ``(x, normed for next_norm or None, latents, weights)``."""
        batch, s, w = x.shape
        rows = x.reshape(batch * s, w)
        h = (normed if normed is not None else self.norm1(x)).reshape(batch * s, w)
        if self.kind == "latent_attention":
            out = self.mixer(h, batch, self.layer_id, self.kv_layer, cache, latent, keep, output_attentions)
        else:
            out = self.mixer(h, batch, self.layer_id, cache, keep)
        after = self.norm2 if self.mlp is not None else next_norm
        rows, h = self._join(rows, out.y, out.side["rg"], self.rg1_bias, self.norm1b, after)
        if self.mlp is not None:
            f = self.mlp(h)
            rows, h = self._join(rows, f.y, f.side["rg"], self.rg2_bias, self.norm2b, next_norm, f.slots, f.weights)
        return rows.view(batch, s, w), (h.view(batch, s, w) if h is not None else None), out.latent, out.probs


_LAYER_KEY = re.compile(r"l(\d+)\.(.+)$")


class MoronexPreTrainedModel(PreTrainedModel):
    config_class = MoronexConfig
    base_model_prefix = "transformer"

    def get_layer_policies(self):
        return [MoronexLayerPolicy]

    def _exec_both_engines(self, tensor_parallel_size: int = 1, pipeline_parallel_size: int = 1, **kw: Any):
        if int(tensor_parallel_size) > 1 or int(pipeline_parallel_size) > 1:
            raise NotImplementedError("Moronex runs on one GPU per replica: its packed projections and shared latents have no "
                                      "tensor- or pipeline-parallel layout (data parallelism works)")
        return super()._exec_both_engines(tensor_parallel_size=1, pipeline_parallel_size=1, **kw)

    def convert_checkpoint(self, state_dict: Dict[str, Tensor]) -> Dict[str, Tensor]:
        """Flat checkpoint names -> module names. Every tensor must be there, with its shape, and none may be left over."""
        if "embed" not in state_dict:
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

        put("wte.weight", model.wte.weight, "embed")
        put("ln_f.weight", model.ln_f.weight, "final.norm")
        for i, b in enumerate(model.h):
            at, mx = f"h.{i}.", f"l{i}.mix."
            for n in ("norm1", "norm1b"):
                put(f"{at}{n}.weight", getattr(b, n).weight, f"l{i}.{n}")
            put(f"{at}rg1_bias", b.rg1_bias, f"l{i}.rg1.b")
            mixer = b.mixer
            parts = {n: take(f"l{i}.rg1" if n == "rg" else mx + n) for n in mixer.in_proj.parts}
            out[f"transformer.{at}mixer.in_proj.weight"] = mixer.in_proj.pack(parts)
            put(f"{at}mixer.out_proj.weight", mixer.out_proj.weight, mx + "o")
            if b.kind == "latent_attention":
                put(f"{at}mixer.q_norm.weight", mixer.q_norm.weight, mx + "dq.norm")
                if mixer.kv_norm is not None:
                    put(f"{at}mixer.kv_norm.weight", mixer.kv_norm.weight, mx + "dkv.norm")
                put(f"{at}mixer.uq.weight", mixer.uq.weight, mx + "uq")
                out[f"transformer.{at}mixer.kv_up.weight"] = mixer.kv_up.pack({"k": take(mx + "uk"), "v": take(mx + "uv")})
                put(f"{at}mixer.sink", mixer.sink, mx + "sink")
            else:
                put(f"{at}mixer.f_bias", mixer.f_bias, mx + "f.b")
                put(f"{at}mixer.lower", mixer.lower, mx + "lower")
                put(f"{at}mixer.o_norm.weight", mixer.o_norm.weight, mx + "norm")
            if b.mlp is None:
                continue
            fw = f"l{i}.mlp."
            for n in ("norm2", "norm2b"):
                put(f"{at}{n}.weight", getattr(b, n).weight, f"l{i}.{n}")
            put(f"{at}rg2_bias", b.rg2_bias, f"l{i}.rg2.b")
            parts = {n: take(f"l{i}.rg2" if n == "rg" else fw + n) for n in b.mlp.in_proj.parts}
            out[f"transformer.{at}mlp.in_proj.weight"] = b.mlp.in_proj.pack(parts)
            if isinstance(b.mlp, GatedMLP):
                put(f"{at}mlp.down.weight", b.mlp.down.weight, fw + "down")
            else:
                put(f"{at}mlp.router.weight", b.mlp.router.weight, fw + "router")
                put(f"{at}mlp.router.bias", b.mlp.router.bias, fw + "router.b")
                for n in ("up", "down"):
                    shape = getattr(b.mlp, n).shape[1:]
                    out[f"transformer.{at}mlp.{n}"] = torch.stack([take(f"{fw}e{e}.{n}", shape) for e in range(b.mlp.experts)])
        head = src.pop("head", None)
        if isinstance(self, MoronexForCausalLM):
            if head is None:
                raise KeyError("checkpoint has no tensor 'head'")
            out["lm_head.weight"] = head
        if src:
            raise KeyError(f"checkpoint tensors that no layer of the configuration uses: {sorted(src)[:8]}")
        return out


class MoronexModel(DecoderBackbone, MoronexPreTrainedModel):
    def __init__(self, config: MoronexConfig) -> None:
        super().__init__(config)
        self.wte = Embedding(config.vocab, config.width)
        self.h = nn.ModuleList([MoronexBlock(config, i) for i in range(len(config.layers))])
        self.ln_f = RMSNorm(config.width, config.eps, offset=1.0)
        self.post_init()

    def embed(self, input_ids, position_ids, token_type_ids, inputs_embeds):
        hs = self.wte(input_ids) if inputs_embeds is None else inputs_embeds
        return hs.to(torch.float32)                        # the residual stream is fp32

    def prepare_fn(self, past_key_values=None, use_cache=None, token_type_ids=None, head_mask=None, **kw):
        if token_type_ids is not None or head_mask is not None:
            raise ValueError("Moronex has neither token types nor head masks")
        use_cache = self.config.use_cache if use_cache is None else use_cache
        if past_key_values is not None and not isinstance(past_key_values, StaticKVCache):
            raise TypeError("Moronex continues from a StaticKVCache (what its outputs return)")
        if past_key_values is None and use_cache and not (self.training and torch.is_grad_enabled()):
            ref = next((kw[k] for k in ("input_ids", "inputs_embeds", "hidden_states") if kw.get(k) is not None), None)
            past_key_values = StaticKVCache(ref.shape[1] if ref is not None and ref.dim() > 1 else 1, grow=True)
        kw = super().prepare_fn(past_key_values=past_key_values, use_cache=use_cache, **kw)
        kw["presents"] = None
        kw["_normed"] = None
        kw["_latents"] = {}
        if kw["attention_mask"] is not None:
            kw["attention_mask"] = (kw["attention_mask"] != 0).to(torch.uint8)
        return kw

    def block_fn(self, layer_id: int, **kw) -> Dict[str, Any]:
        block = self.h[layer_id]
        hs = kw["hidden_states"]
        if kw["all_hidden_states"] is not None:
            kw["all_hidden_states"].append(hs)
        last = layer_id + 1 == len(self.h)
        args = dict(next_norm=self.ln_f if last else self.h[layer_id + 1].norm1, cache=kw["cache"], keep=kw["attention_mask"],
                    output_attentions=kw["output_attentions"])
        latent = kw["_latents"].get(block.kv_layer)
        if self.gradient_checkpointing and self.training and torch.is_grad_enabled():
            hs, normed, own, probs = checkpoint(lambda x, n, c: block(x, n, latent=c, **args), hs, kw["_normed"], latent,
                                                use_reentrant=False)
        else:
            hs, normed, own, probs = block(hs, kw["_normed"], latent=latent, **args)
        if own is not None and block.kv_layer == layer_id:
            kw["_latents"][layer_id] = own
        kw["hidden_states"], kw["_normed"] = hs, normed
        if kw["all_attentions"] is not None:
            kw["all_attentions"].append(probs)
        return kw

    def postblock_fn(self, **kw) -> Dict[str, Any]:
        hs = kw["_normed"] if kw["_normed"] is not None else self.ln_f(kw["hidden_states"])
        if kw["all_hidden_states"] is not None:
            kw["all_hidden_states"].append(kw["hidden_states"])
        if kw["cache"] is not None:
            kw["cache"].advance(kw["_seq"])
        kw["hidden_states"] = hs
        return kw


class MoronexForCausalLM(CausalLMHeadMixin, MoronexPreTrainedModel):
    def __init__(self, config: MoronexConfig) -> None:
        super().__init__(config)
        self.transformer = MoronexModel(config)
        self.lm_head = Linear(config.width, config.vocab, bias=False)
        self.post_init()

    def get_head_layers(self) -> List[Layer]:
        return [Layer(module=self.lm_head, weight=self.lm_head.weight, parallel=False)]


class MoronexForSequenceClassification(SequenceClassificationMixin, MoronexPreTrainedModel):
    def __init__(self, config: MoronexConfig) -> None:
        super().__init__(config)
        self.num_labels = config.num_labels
        self.transformer = MoronexModel(config)
        self.score = Linear(config.width, self.num_labels, bias=False)
        self.post_init()

    def get_head_layers(self) -> List[Layer]:
        return [Layer(module=self.score, weight=self.score.weight, parallel=False)]


class MoronexLayerPolicy(LayerPolicy):
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
        return MoronexBlock
