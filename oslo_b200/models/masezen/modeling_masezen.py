"""Masezen: a decoder whose layers are listed one by one in the configuration, with both sublayers of a layer side by side.

A layer's mixer is grouped-query attention whose heads' scores are mixed before the softmax and whose values are its keys; its
feed-forward is dense (squared relu), a mixture of clamped gated experts whose weights scale what the experts read, or none.
One norm (a single number as its weight) serves both; the mixer reads its result through a short causal convolution:

    h = norm(x);  x <- x + ls1 * mixer(h + conv(h)) + ls2 * ff(h);  x <- x + norm(W_proj (gelu(W_gate x) * e))

where ``e`` is the layer's part of the token's own row in a table beside the embedding. The residual stream is fp32 whatever
the parameter dtype. One kernel adds a layer's sublayers (``ops.branch_join``), a second one the token's part, and writes the next
layer's normed input, across block borders too.

Checkpoints use flat names (``l3.mix.q``, ``l3.mlp.e0.up``, ``l3.canon1``, ...); ``convert_checkpoint`` packs them into the modules.
"""
from __future__ import annotations

from typing import Any, Dict, List, NamedTuple, Optional

import torch
import torch.nn as nn
from torch import Tensor
from torch.utils.checkpoint import checkpoint

from ... import ops
from ...modeling_utils import PretrainedConfig, PreTrainedModel
from ...ops.reference import Branch
from ...parallel.layers import Embedding, Linear, RMSNorm
from ...parallel.mpu import Layer, LayerPolicy
from ...utils.streams import beside
from ..common import CausalLMHeadMixin, DecoderBackbone, SequenceClassificationMixin, StaticKVCache
from ..mixers import DenseMLP, GroupedQueryAttention, InputConvolution, MixtureOfExperts, TokenInput

_MIXER_KEYS = ("heads", "kv_heads", "dim", "vdim", "scale", "rot")
_SCALING_KEYS = ("factor", "original", "fast", "slow")


class MasezenConfig(PretrainedConfig):
    """``layers``: one dictionary per layer with ``type`` (``attention``), the mixer's sizes ``mixer`` (``rot`` with ``dims``, ``base`` and, for
    YaRN, ``scaling``) and the feed-forward ``mlp`` (``{"kind": "dense", "ff": ...}``, ``{"kind": "moe", "expert": {"ff": ..., "limit":
    ...}, "router": {"experts": ..., "top": ...}, "shared": {"ff": ..., "limit": ...}}`` or ``None``); ``norm``: ``{"eps": ...}``; ``canon``:
    ``{"taps": ...}`` of the mixers' input convolution; ``token_side``: ``{"dim": ...}`` of the layers' token inputs."""

    model_type = "masezen"
    attribute_map = {"vocab_size": "vocab", "hidden_size": "width", "n_embd": "width"}

    def __init__(self, layers: Optional[List[Dict[str, Any]]] = None, norm: Optional[Dict[str, Any]] = None,
                 canon: Optional[Dict[str, Any]] = None, token_side: Optional[Dict[str, Any]] = None, vocab: int = 32000,
                 width: int = 1024, initializer_range: float = 0.02, use_cache: bool = True, tie_word_embeddings: bool = False,
                 **kwargs: Any) -> None:
        self.layers = list(layers or [])
        self.norm = dict(norm or {"eps": 1e-6})
        self.canon = dict(canon or {"taps": 4})
        self.token_side = dict(token_side or {"dim": 64})
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
        if int(self.canon["taps"]) < 1 or int(self.token_side["dim"]) < 1:
            raise ValueError(f"a convolution of {self.canon['taps']} taps, token inputs of {self.token_side['dim']} dims")
        for i, layer in enumerate(self.layers):
            kind, m, mlp = layer.get("type"), layer.get("mixer") or {}, layer.get("mlp")
            if kind != "attention":
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            missing = [k for k in _MIXER_KEYS if k not in m]
            if missing:
                raise ValueError(f"layer {i}: {kind} without {missing}")
            if m["heads"] % m["kv_heads"]:
                raise ValueError(f"layer {i}: {m['heads']} query heads over {m['kv_heads']} key / value heads")
            if m["vdim"] != m["dim"]:
                raise ValueError(f"layer {i}: the values are the keys, so vdim {m['vdim']} has to be dim {m['dim']}")
            rot = m["rot"]
            if rot["dims"] % 2 or not 0 <= rot["dims"] <= m["dim"]:
                raise ValueError(f"layer {i}: {rot['dims']} rotated of {m['dim']} dims")
            if rot.get("scaling") is not None and any(k not in rot["scaling"] for k in _SCALING_KEYS):
                raise ValueError(f"layer {i}: rotation scaling needs {_SCALING_KEYS}")
            if mlp is None:
                continue
            if mlp.get("kind") not in ("dense", "moe"):
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            if mlp["kind"] == "moe" and not 1 <= mlp["router"]["top"] <= mlp["router"]["experts"]:
                raise ValueError(f"layer {i}: top {mlp['router']['top']} of {mlp['router']['experts']} experts")


def _mixer(m: Dict[str, Any], width: int, eps: float) -> GroupedQueryAttention:
    rot = m["rot"]
    return GroupedQueryAttention(width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], eps, rot_dims=rot["dims"],
                                 rot_base=rot["base"], rot_scaling=rot.get("scaling"), halves=True, sink=False, value_is_key=True,
                                 gate="element", talk=True)


def _feed_forward(mlp: Optional[Dict[str, Any]], width: int) -> Optional[nn.Module]:
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return DenseMLP(width, mlp["ff"], "relu2")
    expert, router, shared = mlp["expert"], mlp["router"], mlp.get("shared")
    sizes = {} if shared is None else {"shared": shared["ff"], "shared_limit": shared["limit"]}
    return MixtureOfExperts(width, expert["ff"], router["experts"], router["top"], unit="clamped", scored="sigmoid",
                            limit=expert["limit"], scale_input=True, shared_gate=False, **sizes)


class After(NamedTuple):
    """What reads the residual stream after a block: the next block's norm and input convolution, or the final norm."""
    norm: RMSNorm
    canon: Optional[InputConvolution] = None


class MasezenBlock(nn.Module):
    oslo_fused = False

    def __init__(self, config: MasezenConfig, layer_id: int) -> None:
        super().__init__()
        spec, w, eps = config.layers[layer_id], config.width, config.eps
        dim = int(config.token_side["dim"])
        self.layer_id, self.eps = layer_id, eps
        self.norm1 = RMSNorm(None, eps)
        self.canon1 = InputConvolution(w, int(config.canon["taps"]))
        self.mixer = _mixer(spec["mixer"], w, eps)
        self.mlp = _feed_forward(spec.get("mlp"), w)
        self.ls1 = nn.Parameter(torch.ones(w))
        self.ls2 = nn.Parameter(torch.ones(w)) if self.mlp is not None else None
        self.side = TokenInput(w, dim, layer_id * dim, eps)

    def forward(self, x: Tensor, normed: Optional[Tensor], convolved: Optional[Tensor], after: "After", ids: Tensor, table: Tensor,
                cache: Optional[StaticKVCache] = None, keep: Optional[Tensor] = None, positions: Optional[Tensor] = None,
                output_attentions: bool = False):
        """``x`` ``[batch, S, width]`` fp32. ``normed``, ``convolved``: ``x`` through this block's norm, and that through its convolution, when
        the previous block computed them; ``after``: what follows this block; ``ids`` ``[batch * S]`` tokens and ``table`` ``[vocab, *]`` of
        their inputs. Returns ``(x, x through the norm that follows, that through the convolution that follows or None, attention
        weights or None)``."""
        batch, s, w = x.shape
        rows = x.reshape(batch * s, w)
        h = (self.norm1(rows) if normed is None else normed).reshape(batch * s, w)

        def attend():
            c = self.canon1(h, batch, self.layer_id, cache, keep) if convolved is None else convolved
            return self.mixer(c, batch, self.layer_id, cache, keep, positions, output_attentions)

        out, f = beside(attend, lambda: None if self.mlp is None else self.mlp(h), h)
        branches = [Branch(out.y, self.ls1, normed=False)]
        if f is not None:
            top = self.mlp.top if isinstance(self.mlp, MixtureOfExperts) else 0
            branches.append(Branch(f.y, self.ls2, normed=False, slots=f.slots, top=top))
            if f.shared is not None:
                branches.append(Branch(f.shared, self.ls2, normed=False))
        rows, (copy,) = ops.branch_join(rows, branches, 1.0, self.eps, [], copy=self.ls1.dtype, fused=self.oslo_fused)
        conv = None
        if s == 1 and cache is not None and after.canon is not None:          # single tokens: the join does the next convolution too
            conv = after.canon.step(batch, self.layer_id + 1, cache, keep, x.device)
        rows, (h, *more) = ops.branch_join(rows, [self.side(copy, ids, table)], 1.0, self.eps, [after.norm.weight], conv=conv,
                                           fused=self.oslo_fused)
        return rows.view(batch, s, w), h.view(batch, s, w), more[0] if more else None, out.probs


class MasezenPreTrainedModel(PreTrainedModel):
    config_class = MasezenConfig
    base_model_prefix = "transformer"

    def get_layer_policies(self):
        return [MasezenLayerPolicy]

    def _exec_both_engines(self, tensor_parallel_size: int = 1, pipeline_parallel_size: int = 1, **kw: Any):
        if int(tensor_parallel_size) > 1 or int(pipeline_parallel_size) > 1:
            raise NotImplementedError("Masezen runs on one GPU per replica: its packed projections, mixed heads and convolution states "
                                      "have no tensor- or pipeline-parallel layout (data parallelism works)")
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
        put("side_table.weight", model.side_table.weight, "side.embed")
        put("ln_f.weight", model.ln_f.weight, "final.norm")
        for i, b in enumerate(model.h):
            at, mx, fw, mixer, mlp = f"h.{i}.", f"l{i}.mix.", f"l{i}.mlp.", b.mixer, b.mlp
            put(f"{at}norm1.weight", b.norm1.weight, f"l{i}.norm1")
            put(f"{at}canon1.weight", b.canon1.weight, f"l{i}.canon1")
            put(f"{at}ls1", b.ls1, f"l{i}.ls1")
            for n in ("gate", "proj", "norm"):
                put(f"{at}side.{n}.weight", getattr(b.side, n).weight, f"l{i}.side.{n}")
            put_packed(at + "mixer.in_proj", mixer.in_proj, mx)
            put(f"{at}mixer.q_norm.weight", mixer.q_norm.weight, mx + "q.norm")
            put(f"{at}mixer.k_norm.weight", mixer.k_norm.weight, mx + "k.norm")
            put(f"{at}mixer.talk", mixer.talk, mx + "talk")
            put(f"{at}mixer.out_proj.weight", mixer.out_proj.weight, mx + "o")
            if mlp is None:
                continue
            put(f"{at}ls2", b.ls2, f"l{i}.ls2")
            if isinstance(mlp, DenseMLP):
                put(f"{at}mlp.up.weight", mlp.up.weight, fw + "up")
                put(f"{at}mlp.down.weight", mlp.down.weight, fw + "down")
                continue
            put(f"{at}mlp.router.weight", mlp.router.weight, fw + "router")
            n, ff, width = mlp.experts, mlp.down.size(2), mlp.down.size(1)
            out[f"transformer.{at}mlp.up"] = torch.stack([MixtureOfExperts.interleave(
                take(f"{fw}e{e}.gate", (ff, width)), take(f"{fw}e{e}.up", (ff, width))) for e in range(n)])
            out[f"transformer.{at}mlp.down"] = torch.stack([take(f"{fw}e{e}.down", (width, ff)) for e in range(n)])
            if mlp.shared is not None:
                put_packed(at + "mlp.shared.in_proj", mlp.shared.in_proj, fw + "shared.")
                put(f"{at}mlp.shared.down.weight", mlp.shared.down.weight, fw + "shared.down")
        head = src.pop("head", None)
        if isinstance(self, MasezenForCausalLM):
            if head is None:
                raise KeyError("checkpoint has no tensor 'head'")
            out["lm_head.weight"] = head
        if src:
            raise KeyError(f"checkpoint tensors that no layer of the configuration uses: {sorted(src)[:8]}")
        return out


class MasezenModel(DecoderBackbone, MasezenPreTrainedModel):
    def __init__(self, config: MasezenConfig) -> None:
        super().__init__(config)
        self.wte = Embedding(config.vocab, config.width)
        self.side_table = Embedding(config.vocab, len(config.layers) * int(config.token_side["dim"]))
        self.h = nn.ModuleList([MasezenBlock(config, i) for i in range(len(config.layers))])
        self.ln_f = RMSNorm(None, config.eps)
        self.post_init()

    def embed(self, input_ids, position_ids, token_type_ids, inputs_embeds):
        hs = self.wte(input_ids) if inputs_embeds is None else inputs_embeds
        return hs.to(torch.float32)                        # the residual stream is fp32

    def prepare_fn(self, input_ids=None, past_key_values=None, use_cache=None, token_type_ids=None, head_mask=None, **kw):
        if token_type_ids is not None or head_mask is not None:
            raise ValueError("Masezen has neither token types nor head masks")
        if input_ids is None:
            raise ValueError("Masezen's layers read the tokens themselves: input_ids is required")
        use_cache = self.config.use_cache if use_cache is None else use_cache
        if past_key_values is not None and not isinstance(past_key_values, StaticKVCache):
            raise TypeError("Masezen continues from a StaticKVCache (what its outputs return)")
        if past_key_values is None and use_cache and not (self.training and torch.is_grad_enabled()):
            past_key_values = StaticKVCache(input_ids.shape[-1], grow=True)
        kw = super().prepare_fn(input_ids=input_ids, past_key_values=past_key_values, use_cache=use_cache, **kw)
        kw["presents"] = None
        kw["_normed"] = kw["_convolved"] = None
        kw["_ids"] = kw["input_ids"].reshape(-1)
        if kw["attention_mask"] is not None:
            kw["attention_mask"] = (kw["attention_mask"] != 0).to(torch.uint8)
        return kw

    def block_fn(self, layer_id: int, **kw) -> Dict[str, Any]:
        block = self.h[layer_id]
        hs = kw["hidden_states"]
        if kw["all_hidden_states"] is not None:
            kw["all_hidden_states"].append(hs)
        after = After(self.ln_f) if layer_id + 1 == len(self.h) else After(self.h[layer_id + 1].norm1, self.h[layer_id + 1].canon1)
        args = dict(convolved=kw["_convolved"], after=after, ids=kw["_ids"], table=self.side_table.weight, cache=kw["cache"], keep=kw["attention_mask"],
                    positions=kw["position_ids"], output_attentions=kw["output_attentions"])
        if self.gradient_checkpointing and self.training and torch.is_grad_enabled():
            hs, normed, convolved, probs = checkpoint(lambda x, n: block(x, n, **args), hs, kw["_normed"], use_reentrant=False)
        else:
            hs, normed, convolved, probs = block(hs, kw["_normed"], **args)
        kw["hidden_states"], kw["_normed"], kw["_convolved"] = hs, normed, convolved
        if kw["all_attentions"] is not None:
            kw["all_attentions"].append(probs)
        return kw

    def postblock_fn(self, **kw) -> Dict[str, Any]:
        hs = self.ln_f(kw["hidden_states"]) if kw["_normed"] is None else kw["_normed"]
        if kw["all_hidden_states"] is not None:
            kw["all_hidden_states"].append(kw["hidden_states"])
        if kw["cache"] is not None:
            kw["cache"].advance(kw["_seq"])
        kw["hidden_states"] = hs
        return kw


class MasezenForCausalLM(CausalLMHeadMixin, MasezenPreTrainedModel):
    def __init__(self, config: MasezenConfig) -> None:
        super().__init__(config)
        self.transformer = MasezenModel(config)
        self.lm_head = Linear(config.width, config.vocab, bias=False)
        self.post_init()

    def get_head_layers(self) -> List[Layer]:
        return [Layer(module=self.lm_head, weight=self.lm_head.weight, parallel=False)]


class MasezenForSequenceClassification(SequenceClassificationMixin, MasezenPreTrainedModel):
    def __init__(self, config: MasezenConfig) -> None:
        super().__init__(config)
        self.num_labels = config.num_labels
        self.transformer = MasezenModel(config)
        self.score = Linear(config.width, self.num_labels, bias=False)
        self.post_init()

    def get_head_layers(self) -> List[Layer]:
        return [Layer(module=self.score, weight=self.score.weight, parallel=False)]


class MasezenLayerPolicy(LayerPolicy):
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
        return MasezenBlock
