"""Dekutar: a decoder whose layers are listed one by one in the configuration, on several residual streams.

A layer is a mixer - ``attention`` (grouped-query attention whose values are its keys, in a sliding window that keeps the first
tokens), ``latent_attention`` (low-rank latents with a rotated key part) or ``mlstm`` (matrix memory) - and a mixture of experts (or
none). Both sublayers read a weighted sum of the streams through a norm, and every stream becomes a mix of the old ones plus
its share of the result:

    u = sum_s in[s] x_s;  y = sublayer(norm(u));  x_t <- sum_s mix[s, t] x_s + out[t] y

with the streams in fp32 whatever the parameter dtype. One kernel per sublayer adds up the experts' rows, updates the streams
and writes the next sublayer's normed input (``ops.hyper_join``), across block borders too. ``hidden_states`` between blocks is
``[batch, S, streams, width]``; what the model returns is the sum of the streams.

Checkpoints use flat names (``l3.mix.q``, ``l3.mlp.e0.up``, ``l3.hc1.mix``, ...); ``convert_checkpoint`` packs them into the modules.
"""
from __future__ import annotations

from typing import Any, Dict, List, NamedTuple, Optional

import torch
import torch.nn as nn
from torch import Tensor
from torch.utils.checkpoint import checkpoint

from ... import ops
from ...modeling_utils import PretrainedConfig, PreTrainedModel
from ...ops.reference import SublayerResult
from ...parallel.layers import Embedding, Linear, RMSNorm
from ...parallel.mpu import Layer, LayerPolicy
from ..common import CausalLMHeadMixin, DecoderBackbone, SequenceClassificationMixin, StaticKVCache
from ..mixers import GroupedQueryAttention, HyperConnections, LatentAttention, MatrixMemory, MixtureOfExperts

_MIXER_KEYS = {
    "attention": ("heads", "kv_heads", "dim", "vdim", "scale", "mask", "rot"),
    "latent_attention": ("heads", "dim", "vdim", "rot_dim", "q_rank", "kv_rank", "scale", "rot"),
    "mlstm": ("heads", "dim", "vdim", "gate_cap"),
}
MAX_STREAMS = 16   # residual streams that the join kernel covers


class DekutarConfig(PretrainedConfig):
    """``layers``: one dictionary per layer with ``type`` (``attention`` | ``latent_attention`` | ``mlstm``), the mixer's sizes ``mixer`` and
    the feed-forward ``mlp`` (``{"kind": "moe", "expert": {"ff": ...}, "router": {"experts": ..., "identity": ..., "top": ...},
    "shared": {"ff": ...}}`` or ``None``); ``embedding``: ``{"scale": ...}``; ``norm``: ``{"eps": ...}``; ``streams``; ``logit_scale``."""

    model_type = "dekutar"
    attribute_map = {"vocab_size": "vocab", "hidden_size": "width", "n_embd": "width"}

    def __init__(self, layers: Optional[List[Dict[str, Any]]] = None, norm: Optional[Dict[str, Any]] = None,
                 embedding: Optional[Dict[str, Any]] = None, streams: int = 1, logit_scale: float = 1.0, vocab: int = 32000,
                 width: int = 1024, initializer_range: float = 0.02, use_cache: bool = True, tie_word_embeddings: bool = False,
                 **kwargs: Any) -> None:
        self.layers = list(layers or [])
        self.norm = dict(norm or {"eps": 1e-6})
        self.embedding = dict(embedding or {"scale": 1.0})
        self.streams, self.logit_scale = int(streams), float(logit_scale)
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
        if not 1 <= self.streams <= MAX_STREAMS:
            raise ValueError(f"{self.streams} residual streams (1 to {MAX_STREAMS})")
        for i, layer in enumerate(self.layers):
            kind, m, mlp = layer.get("type"), layer.get("mixer") or {}, layer.get("mlp")
            if kind not in _MIXER_KEYS:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            missing = [k for k in _MIXER_KEYS[kind] if k not in m]
            if missing:
                raise ValueError(f"layer {i}: {kind} without {missing}")
            if kind == "attention":
                if m["heads"] % m["kv_heads"]:
                    raise ValueError(f"layer {i}: {m['heads']} query heads over {m['kv_heads']} key / value heads")
                if m["vdim"] != m["dim"]:
                    raise ValueError(f"layer {i}: the values are the keys, so vdim {m['vdim']} has to be dim {m['dim']}")
                if m["rot"]["dims"] % 2 or not 0 <= m["rot"]["dims"] <= m["dim"]:
                    raise ValueError(f"layer {i}: {m['rot']['dims']} rotated of {m['dim']} dims")
                if m["mask"]["size"] < 1 or m["mask"]["keep_first"] < 0:
                    raise ValueError(f"layer {i}: a window of {m['mask']['size']} with {m['mask']['keep_first']} first tokens")
            if kind == "latent_attention" and (m["rot_dim"] % 2 or m["rot"]["dims"] != m["rot_dim"]):
                raise ValueError(f"layer {i}: {m['rot']['dims']} rotated of {m['rot_dim']} rotary dims")
            if mlp is None:
                continue
            if mlp.get("kind") != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            r = mlp["router"]
            if not 1 <= r["top"] <= r["experts"] + r.get("identity", 0):
                raise ValueError(f"layer {i}: top {r['top']} of {r['experts']} + {r.get('identity', 0)} experts")


def _mixer(kind: str, m: Dict[str, Any], width: int, eps: float) -> nn.Module:
    if kind == "attention":
        return GroupedQueryAttention(width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], eps, rot_dims=m["rot"]["dims"],
                                     rot_base=m["rot"]["base"], norm_weights=False, sink=False, window=m["mask"]["size"],
                                     keep_first=m["mask"]["keep_first"], value_is_key=True, gate="head")
    if kind == "latent_attention":
        return LatentAttention(width, m["heads"], m["dim"], m["vdim"], m["q_rank"], m["kv_rank"], m["scale"], eps, rot_dim=m["rot_dim"],
                               rot_base=m["rot"]["base"], sink=False, gate="element")
    return MatrixMemory(width, m["heads"], m["dim"], m["vdim"], m["gate_cap"], eps)


class NextInput(NamedTuple):
    """How the sublayer after this one reads the streams."""
    w_in: Optional[Tensor]                 # None: their plain sum
    norm: RMSNorm
    scale: float = 1.0


class DekutarBlock(nn.Module):
    oslo_fused = False

    def __init__(self, config: DekutarConfig, layer_id: int) -> None:
        super().__init__()
        spec, w, eps = config.layers[layer_id], config.width, config.eps
        mlp = spec.get("mlp")
        self.kind, self.layer_id = spec["type"], layer_id
        self.norm1 = RMSNorm(w, eps, offset=1.0)
        self.hc1 = HyperConnections(config.streams)
        self.mixer = _mixer(self.kind, spec["mixer"], w, eps)
        self.norm2 = self.hc2 = self.mlp = None
        if mlp is not None:
            self.norm2 = RMSNorm(w, eps, offset=1.0)
            self.hc2 = HyperConnections(config.streams)
            router, shared = mlp["router"], mlp.get("shared")
            self.mlp = MixtureOfExperts(w, mlp["expert"]["ff"], router["experts"], router["top"], unit="silu", scored=True,
                                        identity=router.get("identity", 0), shared=None if shared is None else shared["ff"])

    def reads(self) -> NextInput:
        return NextInput(self.hc1.w_in, self.norm1)

    def forward(self, x: Tensor, normed: Optional[Tensor], after: NextInput, cache: Optional[StaticKVCache] = None,
                keep: Optional[Tensor] = None, positions: Optional[Tensor] = None, lead: Optional[Tensor] = None,
                output_attentions: bool = False):
        """``x`` ``[batch, S, streams, width]`` fp32. ``normed``: this block's input read from ``x`` when the previous block did that;
        ``after``: what follows this block. Returns ``(x, the input of what follows, attention weights or None)``."""
        batch, s, n, w = x.shape
        rows = x.view(batch * s, n, w) if x.is_contiguous() else x.flatten(0, 1)
        if normed is None:
            _, normed = self.hc1(rows, None, *self.reads())
        h = normed.reshape(batch * s, w)
        if self.kind == "attention":
            out = self.mixer(h, batch, self.layer_id, cache, keep, positions, output_attentions, lead)
        elif self.kind == "latent_attention":
            out = self.mixer(h, batch, self.layer_id, self.layer_id, cache, None, keep, output_attentions, positions)
        else:
            out = self.mixer(h, batch, self.layer_id, cache, keep)
        rows, h = self.hc1(rows, SublayerResult(out.y), *(after if self.mlp is None else NextInput(self.hc2.w_in, self.norm2)))
        if self.mlp is not None:
            f = self.mlp(h)
            result = SublayerResult(f.y, f.slots, f.weights, f.choice, self.mlp.experts, h, f.shared, f.shared_gate)
            rows, h = self.hc2(rows, result, *after)
        return rows.view(batch, s, n, w), h.view(batch, s, w), out.probs


class DekutarPreTrainedModel(PreTrainedModel):
    config_class = DekutarConfig
    base_model_prefix = "transformer"

    def get_layer_policies(self):
        return [DekutarLayerPolicy]

    def _exec_both_engines(self, tensor_parallel_size: int = 1, pipeline_parallel_size: int = 1, **kw: Any):
        if int(tensor_parallel_size) > 1 or int(pipeline_parallel_size) > 1:
            raise NotImplementedError("Dekutar runs on one GPU per replica: its packed projections and recurrent states have no "
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

        def put_packed(name: str, packed, source: str) -> None:
            out[f"transformer.{name}.weight"] = packed.pack({n: take(source + n) for n in packed.parts})

        put("wte.weight", model.wte.weight, "embed")
        put("ln_f.weight", model.ln_f.weight, "final.norm")
        for i, b in enumerate(model.h):
            at, mx, fw, mixer = f"h.{i}.", f"l{i}.mix.", f"l{i}.mlp.", b.mixer
            mat = at + "mixer."
            for which in ("1", "2") if b.mlp is not None else ("1",):
                put(f"{at}norm{which}.weight", getattr(b, "norm" + which).weight, f"l{i}.norm{which}")
                for n in ("in", "out"):
                    put(f"{at}hc{which}.w_{n}", getattr(getattr(b, "hc" + which), "w_" + n), f"l{i}.hc{which}.{n}")
                put(f"{at}hc{which}.mix", getattr(b, "hc" + which).mix, f"l{i}.hc{which}.mix")
            put_packed(mat + "in_proj", mixer.in_proj, mx)
            put(f"{mat}out_proj.weight", mixer.out_proj.weight, mx + "o")
            if b.kind == "latent_attention":
                put(f"{mat}q_norm.weight", mixer.q_norm.weight, mx + "dq.norm")
                put(f"{mat}kv_norm.weight", mixer.kv_norm.weight, mx + "dkv.norm")
                put(f"{mat}uq.weight", mixer.uq.weight, mx + "uq")
                put_packed(mat + "kv_up", mixer.kv_up, mx + "u")
            elif b.kind == "mlstm":
                heads, width = mixer.heads, mixer.in_proj.in_features
                out[f"transformer.{mat}gates.weight"] = torch.cat([take(mx + n, (heads, width)) for n in ("i", "f")])
                out[f"transformer.{mat}gates.bias"] = torch.cat([take(f"{mx}{n}.b", (heads,)) for n in ("i", "f")])
                put(f"{mat}o_norm", mixer.o_norm, mx + "norm")
            if b.mlp is None:
                continue
            put(f"{at}mlp.router.weight", b.mlp.router.weight, fw + "router")
            put(f"{at}mlp.correction", b.mlp.correction, fw + "correction")
            n, ff, width = b.mlp.experts, b.mlp.down.size(2), b.mlp.down.size(1)
            if n:
                out[f"transformer.{at}mlp.up"] = torch.stack([MixtureOfExperts.interleave(
                    take(f"{fw}e{e}.gate", (ff, width)), take(f"{fw}e{e}.up", (ff, width))) for e in range(n)])
                out[f"transformer.{at}mlp.down"] = torch.stack([take(f"{fw}e{e}.down", (width, ff)) for e in range(n)])
            if b.mlp.shared is not None:
                put_packed(at + "mlp.shared.in_proj", b.mlp.shared.in_proj, fw + "shared.")
                put(f"{at}mlp.shared.down.weight", b.mlp.shared.down.weight, fw + "shared.down")
        head = src.pop("head", None)
        if isinstance(self, DekutarForCausalLM):
            if head is None:
                raise KeyError("checkpoint has no tensor 'head'")
            out["lm_head.weight"] = head
        if src:
            raise KeyError(f"checkpoint tensors that no layer of the configuration uses: {sorted(src)[:8]}")
        return out


class DekutarModel(DecoderBackbone, DekutarPreTrainedModel):
    """``output_scale``: factor on the final norm's result (a causal LM's ``logit_scale``, which saves a pass over the logits)."""

    def __init__(self, config: DekutarConfig, output_scale: float = 1.0) -> None:
        super().__init__(config)
        self.output_scale = float(output_scale)
        self.wte = Embedding(config.vocab, config.width)
        self.h = nn.ModuleList([DekutarBlock(config, i) for i in range(len(config.layers))])
        self.ln_f = RMSNorm(config.width, config.eps, offset=1.0)
        self.post_init()

    def embed(self, input_ids, position_ids, token_type_ids, inputs_embeds):
        hs = self.wte(input_ids) if inputs_embeds is None else inputs_embeds
        hs = hs.to(torch.float32) * float(self.config.embedding["scale"])        # the residual streams are fp32
        return hs.unsqueeze(2).expand(-1, -1, self.config.streams, -1)           # all equal: no copy until a sublayer writes them

    def prepare_fn(self, past_key_values=None, use_cache=None, token_type_ids=None, head_mask=None, **kw):
        if token_type_ids is not None or head_mask is not None:
            raise ValueError("Dekutar has neither token types nor head masks")
        use_cache = self.config.use_cache if use_cache is None else use_cache
        if past_key_values is not None and not isinstance(past_key_values, StaticKVCache):
            raise TypeError("Dekutar continues from a StaticKVCache (what its outputs return)")
        if past_key_values is None and use_cache and not (self.training and torch.is_grad_enabled()):
            ref = next((kw[k] for k in ("input_ids", "inputs_embeds", "hidden_states") if kw.get(k) is not None), None)
            past_key_values = StaticKVCache(ref.shape[1] if ref is not None and ref.dim() > 1 else 1, grow=True)
        kw = super().prepare_fn(past_key_values=past_key_values, use_cache=use_cache, **kw)
        kw["presents"] = None
        kw["_normed"] = kw["_lead"] = None
        if kw["attention_mask"] is not None:
            kw["attention_mask"] = (kw["attention_mask"] != 0).to(torch.uint8)
            if any(block.kind == "attention" for block in self.h):               # windows keep the first real tokens
                kw["_lead"] = (kw["attention_mask"].cumsum(-1) == 0).sum(-1, dtype=torch.int32)
        return kw

    def block_fn(self, layer_id: int, **kw) -> Dict[str, Any]:
        block = self.h[layer_id]
        hs = kw["hidden_states"]
        if kw["all_hidden_states"] is not None:
            kw["all_hidden_states"].append(hs.sum(2))
        last = layer_id + 1 == len(self.h)
        args = dict(after=NextInput(None, self.ln_f, self.output_scale) if last else self.h[layer_id + 1].reads(), cache=kw["cache"],
                    keep=kw["attention_mask"], positions=kw["position_ids"], lead=kw["_lead"], output_attentions=kw["output_attentions"])
        if self.gradient_checkpointing and self.training and torch.is_grad_enabled():
            hs, normed, probs = checkpoint(lambda x, n: block(x, n, **args), hs, kw["_normed"], use_reentrant=False)
        else:
            hs, normed, probs = block(hs, kw["_normed"], **args)
        kw["hidden_states"], kw["_normed"] = hs, normed
        if kw["all_attentions"] is not None:
            kw["all_attentions"].append(probs)
        return kw

    def postblock_fn(self, **kw) -> Dict[str, Any]:
        hs = kw["_normed"]
        if hs is None:                                     # no blocks
            x = kw["hidden_states"]
            _, hs = ops.hyper_join(x.flatten(0, 1), None, None, None, None, self.ln_f.weight, self.ln_f.eps, self.output_scale,
                                   fused=self.ln_f.oslo_fused)
            hs = hs.view(x.size(0), x.size(1), -1)
        if kw["all_hidden_states"] is not None:
            kw["all_hidden_states"].append(kw["hidden_states"].sum(2))
        if kw["cache"] is not None:
            kw["cache"].advance(kw["_seq"])
        kw["hidden_states"] = hs
        return kw


class DekutarForCausalLM(CausalLMHeadMixin, DekutarPreTrainedModel):
    def __init__(self, config: DekutarConfig) -> None:
        super().__init__(config)
        self.transformer = DekutarModel(config, output_scale=config.logit_scale)
        self.lm_head = Linear(config.width, config.vocab, bias=False)
        self.post_init()

    def get_head_layers(self) -> List[Layer]:
        return [Layer(module=self.lm_head, weight=self.lm_head.weight, parallel=False)]


class DekutarForSequenceClassification(SequenceClassificationMixin, DekutarPreTrainedModel):
    def __init__(self, config: DekutarConfig) -> None:
        super().__init__(config)
        self.num_labels = config.num_labels
        self.transformer = DekutarModel(config)
        self.score = Linear(config.width, self.num_labels, bias=False)
        self.post_init()

    def get_head_layers(self) -> List[Layer]:
        return [Layer(module=self.score, weight=self.score.weight, parallel=False)]


class DekutarLayerPolicy(LayerPolicy):
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
        return DekutarBlock
