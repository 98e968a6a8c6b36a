"""Fedolorn: a decoder-only model with chunked, position-free, output-gated attention and squared-ReLU feed-forwards, some of
them mixtures of experts.

Every layer describes itself (``FedolornLayerConfig``), so sizes, chunk lengths and the kind of feed-forward may change from layer
to layer.  With the residual stream ``x`` in fp32 and ``N`` an RMS norm with weight ``1 + w``:

* ``x = s E[token]``; then per layer ``x += A(N1(x))`` and, unless the layer has no feed-forward, ``x += F(N2(x))``; logits are
  ``N(x) E^T`` with the unscaled embedding ``E``.
* ``A``: grouped-query attention without positions.  A query sees earlier keys of its own chunk of positions; the concatenated
  heads are multiplied by ``sigmoid(W_g h)`` before the output projection.  Key and value sizes are independent.
* ``F``: ``W_down relu(W_up h)^2``, or a mixture of such experts: the router scores experts by a sigmoid, chooses by score plus a
  learned correction within the best groups of neighbouring experts, and weighs by the plain score times a constant.

Serving follows the other models' path (``decode`` over packed tokens and a paged cache); its steps are the attention module's
paged form, the stream kernels of ``ops.residual_stream`` and the expert kernels of ``ops.moe``."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple, Type, Union

import torch
import torch.nn as nn
from torch.utils.checkpoint import checkpoint

from ..compat.hf_checkpoints import HFCheckpointConverter, HFCompatConfig
from ..layers.attention import Attention, AttentionBackend, AttentionConfig, AttentionMask
from ..layers.normalization import LayerNormConfigBase
from ..nn import Embedding, Linear, trunc_normal_
from ..ops import moe
from ..ops.residual_stream import _kernels, add_linear, embed_stream, project
from ..utils.remat import ScanCheckpointPolicy, should_recompute
from .gemma import GemmaNormConfig
from .llama import LlamaLMHeadModel
from .lm_model import LmConfig


@dataclass(frozen=True)
class FedolornLayerConfig:
    """Sizes of one layer.  ``intermediate_dim`` is the feed-forward's (an expert's, when ``num_experts > 0``); None: the layer has
    no feed-forward."""

    num_heads: int = 32
    num_kv_heads: int = 8
    head_dim: int = 128
    v_head_dim: int = 128
    attention_scale: float = 128 ** -0.5
    chunk_size: int = 8192
    intermediate_dim: Optional[int] = 14336
    num_experts: int = 0
    num_experts_per_tok: int = 0
    expert_groups: int = 1
    expert_groups_kept: int = 1
    router_scale: float = 1.0

    def __post_init__(self):
        if self.num_heads % self.num_kv_heads != 0:
            raise ValueError(f"{self.num_heads} query heads cannot share {self.num_kv_heads} key/value heads")
        if self.chunk_size <= 0:
            raise ValueError("chunk_size must be positive")
        if self.num_experts > 0:
            if self.intermediate_dim is None:
                raise ValueError("experts need an intermediate_dim")
            if self.num_experts % self.expert_groups != 0:
                raise ValueError(f"{self.num_experts} experts do not form {self.expert_groups} equal groups")
            if not 0 < self.expert_groups_kept <= self.expert_groups:
                raise ValueError(f"cannot keep {self.expert_groups_kept} of {self.expert_groups} expert groups")
            if not 0 < self.num_experts_per_tok <= self.expert_groups_kept * (self.num_experts // self.expert_groups):
                raise ValueError(f"{self.num_experts_per_tok} experts per token do not fit the kept groups")


def _layer_from_checkpoint(entry: dict) -> FedolornLayerConfig:
    if entry["type"] != "attention":
        raise ValueError(f"unknown layer type {entry['type']!r}")
    m, f = entry["mixer"], entry.get("mlp")
    kw = dict(num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], v_head_dim=m["vdim"], attention_scale=float(m["scale"]),
              chunk_size=m["mask"]["size"], intermediate_dim=None)
    if f is not None:
        if f["kind"] == "dense":
            kw["intermediate_dim"] = f["ff"]
        elif f["kind"] == "moe":
            r = f["router"]
            g = r.get("groups") or {"count": 1, "keep": 1}
            kw.update(intermediate_dim=f["expert"]["ff"], num_experts=r["experts"], num_experts_per_tok=r["top"], expert_groups=g["count"],
                      expert_groups_kept=g["keep"], router_scale=float(r["scale"]))
        else:
            raise ValueError(f"unknown feed-forward kind {f['kind']!r}")
    return FedolornLayerConfig(**kw)


def _layer_to_checkpoint(c: FedolornLayerConfig) -> dict:
    mixer = dict(heads=c.num_heads, kv_heads=c.num_kv_heads, dim=c.head_dim, vdim=c.v_head_dim, scale=c.attention_scale, mask={"size": c.chunk_size})
    if c.intermediate_dim is None:
        mlp = None
    elif c.num_experts == 0:
        mlp = dict(kind="dense", ff=c.intermediate_dim)
    else:
        mlp = dict(kind="moe", expert={"ff": c.intermediate_dim},
                   router=dict(experts=c.num_experts, top=c.num_experts_per_tok, scale=c.router_scale,
                               groups={"count": c.expert_groups, "keep": c.expert_groups_kept}))
    return dict(type="attention", mixer=mixer, mlp=mlp)


@LmConfig.register_subclass("fedolorn")
@dataclass(frozen=True)
class FedolornConfig(HFCompatConfig):
    seq_len: int = 8192
    hidden_dim: int = 4096
    embedding_scale: float = 1.0
    layer_norm_epsilon: float = 1e-5
    layers: Tuple[FedolornLayerConfig, ...] = (FedolornLayerConfig(),)
    initializer_range: float = 0.02
    upcast_attn: bool = False
    attn_backend: Optional[AttentionBackend] = None
    gradient_checkpointing: Union[bool, ScanCheckpointPolicy, str] = True
    reference_checkpoint: Optional[str] = None
    tokenizer: Optional[str] = None
    cross_entropy_block_size: Optional[int] = None

    hf_architecture = "Fedolorn"
    hf_vocab_key = "vocab"
    tie_word_embeddings = True

    def __post_init__(self):
        object.__setattr__(self, "layers", tuple(FedolornLayerConfig(**l) if isinstance(l, dict) else l for l in self.layers))

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def model_type(self) -> Type["FedolornLMHeadModel"]:
        return FedolornLMHeadModel

    def hf_checkpoint_converter(self, ref_checkpoint: Optional[str] = None) -> HFCheckpointConverter:
        return HFCheckpointConverter(self.__class__, reference_checkpoint=ref_checkpoint or self.reference_checkpoint,
                                     tokenizer=ref_checkpoint if self.tokenizer is None else self.tokenizer)

    @classmethod
    def from_hf_config(cls, hf_config) -> "FedolornConfig":
        c = hf_config if isinstance(hf_config, dict) else vars(hf_config)
        return cls(hidden_dim=c["width"], embedding_scale=float(c["embedding"]["scale"]), layer_norm_epsilon=float(c["norm"]["eps"]),
                   layers=tuple(_layer_from_checkpoint(l) for l in c["layers"]))

    def to_hf_config(self, vocab_size: int, config_overrides: Optional[Dict] = None) -> dict:
        cfg = dict(architecture=self.hf_architecture, vocab=vocab_size, width=self.hidden_dim, embedding={"scale": self.embedding_scale},
                   norm={"eps": self.layer_norm_epsilon}, layers=[_layer_to_checkpoint(l) for l in self.layers])
        cfg.update(config_overrides or {})
        return cfg

    @property
    def norm_config(self) -> LayerNormConfigBase:
        return GemmaNormConfig(eps=self.layer_norm_epsilon, use_weight=True, use_bias=False)

    def mk_LayerNorm(self, dim: int):
        return self.norm_config.build(dim)

    def attention_config(self, layer: FedolornLayerConfig) -> AttentionConfig:
        return AttentionConfig(hidden_dim=self.hidden_dim, num_heads=layer.num_heads, num_kv_heads=layer.num_kv_heads, head_dim=layer.head_dim,
                               v_head_dim=layer.v_head_dim, scaling_factor=layer.attention_scale, attention_chunk_size=layer.chunk_size,
                               output_gate=True, upcast_attn=self.upcast_attn, attn_backend=self.attn_backend)

    def _layer_params(self, l: FedolornLayerConfig, active: bool) -> int:
        e = self.hidden_dim
        n = e * (l.num_heads * (l.head_dim + 2 * l.v_head_dim) + l.num_kv_heads * (l.head_dim + l.v_head_dim))
        if l.intermediate_dim is None:
            return n
        if l.num_experts == 0:
            return n + 2 * e * l.intermediate_dim
        return n + e * l.num_experts + 2 * e * l.intermediate_dim * (l.num_experts_per_tok if active else l.num_experts)

    def flops_per_token(self, vocab_size: int) -> float:
        attn = sum(2 * l.num_heads * (l.head_dim + l.v_head_dim) * min(l.chunk_size, self.seq_len) for l in self.layers)
        return 2.0 * (sum(self._layer_params(l, True) for l in self.layers) + vocab_size * self.hidden_dim) + attn

    def total_trainable_params(self, vocab_size: int) -> int:
        e = self.hidden_dim
        extra = sum((e if l.intermediate_dim is None else 2 * e) + l.num_experts for l in self.layers)
        return sum(self._layer_params(l, False) for l in self.layers) + extra + e + vocab_size * e


class SquaredReluMlp(nn.Module):
    """``down(relu(up(x))^2)``."""

    def __init__(self, hidden: int, intermediate: int, *, init_std: float = 0.02):
        super().__init__()
        self.up_proj = Linear(hidden, intermediate, init_std=init_std)
        self.down_proj = Linear(intermediate, hidden, init_std=init_std)

    def add_to_stream(self, stream: torch.Tensor, h: torch.Tensor, batch_info=None) -> torch.Tensor:
        """``stream + mlp(h)``: the activation is applied in the epilogue of the first product, the add in that of the second."""
        if type(self.up_proj) is Linear and type(self.down_proj) is Linear:
            return add_linear(stream, project(h, self.up_proj.weight, squared_relu=True), self.down_proj.weight)
        return stream + self.down_proj(torch.relu(self.up_proj(h)).square()).float()  # wrapped projections (LoRA, fp8)


class SquaredReluExperts(nn.Module):
    """Expert weights ``up [E, ff, hidden]`` and ``down [E, hidden, ff]``."""

    def __init__(self, num_experts: int, hidden: int, intermediate: int, init_std: float):
        super().__init__()
        self.up = nn.Parameter(torch.empty(num_experts, intermediate, hidden))
        self.down = nn.Parameter(torch.empty(num_experts, hidden, intermediate))
        for w in (self.up, self.down):
            if w.device.type != "meta":
                trunc_normal_(w, init_std)
            w.lev_shape = tuple(w.shape)


class GroupedSigmoidMoe(nn.Module):
    """Mixture of squared-ReLU experts with a sigmoid router that chooses within groups of neighbouring experts."""

    def __init__(self, hidden: int, layer: FedolornLayerConfig, *, init_std: float = 0.02):
        super().__init__()
        self.layer = layer
        self.router = Linear(hidden, layer.num_experts, init_std=init_std)
        self.correction = nn.Parameter(torch.zeros(layer.num_experts))  # joins the choice, not the weights
        self.correction.lev_shape = (layer.num_experts,)
        self.experts = SquaredReluExperts(layer.num_experts, hidden, layer.intermediate_dim, init_std)

    def add_to_stream(self, stream: torch.Tensor, h: torch.Tensor, batch_info=None) -> torch.Tensor:
        """``stream + moe(h)``.  ``batch_info``: padding tokens of a packed batch (no cache destination) are sent to no expert."""
        c, e = self.layer, self.experts
        shape = h.shape
        h2 = h.reshape(-1, shape[-1])
        z = project(h2, self.router.weight, out_dtype=torch.float32)
        route = dict(groups=c.expert_groups, keep=c.expert_groups_kept, scale=c.router_scale)
        if _kernels(h2, stream):
            live, limit = (None, 0) if batch_info is None else (batch_info.new_token_dests, batch_info.num_slots)
            routed = moe.route_sigmoid(z, self.correction, c.num_experts_per_tok, live=live, live_limit=limit, **route)
            return moe.add_expert_outputs(stream.view(-1, shape[-1]), h2, routed, e.up, e.down).view(shape)
        idx, w = moe.route_sigmoid_reference(z, self.correction, c.num_experts_per_tok, c.expert_groups, c.expert_groups_kept, c.router_scale)
        return stream + moe.expert_outputs(h2, idx, w, e.up, e.down).view(shape)


class FedolornDecoderLayer(nn.Module):
    """``x`` is the fp32 stream; the norms hand the compute dtype to attention and feed-forward."""

    def __init__(self, config: FedolornConfig, layer: FedolornLayerConfig):
        super().__init__()
        std = config.initializer_range
        self.self_attn = Attention(config.attention_config(layer), init_std=std)
        self.input_layernorm = config.mk_LayerNorm(config.hidden_dim)
        self.mlp = None
        if layer.intermediate_dim is not None:
            self.post_attention_layernorm = config.mk_LayerNorm(config.hidden_dim)
            self.mlp = SquaredReluMlp(config.hidden_dim, layer.intermediate_dim, init_std=std) if layer.num_experts == 0 \
                else GroupedSigmoidMoe(config.hidden_dim, layer, init_std=std)

    def _feed_forward(self, x, batch_info=None):
        if self.mlp is None:
            return x
        return self.mlp.add_to_stream(x, self.post_attention_layernorm.from_stream(x), batch_info)

    def forward(self, x, mask=None, pos_ids=None):
        x = x + self.self_attn(self.input_layernorm.from_stream(x), mask, pos_ids).float()
        return self._feed_forward(x)

    def decode(self, x, kv_cache, batch_info, pos_ids):
        x, kv_cache = self.self_attn.paged_decode_stream(self.input_layernorm.from_stream(x), kv_cache, batch_info, pos_ids, x)
        return self._feed_forward(x, batch_info), kv_cache


class FedolornTransformer(nn.Module):
    def __init__(self, config: FedolornConfig):
        super().__init__()
        self.config = config
        self.layers = nn.ModuleList([FedolornDecoderLayer(config, l) for l in config.layers])
        self.norm = config.mk_LayerNorm(config.hidden_dim)

    def forward(self, x, mask=None, pos_ids=None):
        remat = should_recompute(self.config.gradient_checkpointing) and torch.is_grad_enabled() and self.training
        for layer in self.layers:
            x = checkpoint(layer, x, mask, pos_ids, use_reentrant=False) if remat else layer(x, mask, pos_ids)
        return self.norm.from_stream(x)

    def decode(self, x, caches, batch_info, pos_ids, logit_rows=None):
        new = []
        for layer, c in zip(self.layers, caches):
            x, c = layer.decode(x, c, batch_info, pos_ids)
            new.append(c)
        return self.norm.from_stream(x, rows=logit_rows), new

    def initial_cache(self, max_pages: int, page_size: int, *, dtype=torch.bfloat16, device=None):
        return [l.self_attn.empty_page_cache(max_pages, page_size, dtype=dtype, device=device) for l in self.layers]


class FedolornEmbedding(nn.Module):
    def __init__(self, vocab_size: int, config: FedolornConfig):
        super().__init__()
        self.scale = config.embedding_scale
        self.token_embeddings = Embedding(vocab_size, config.hidden_dim, init_std=config.initializer_range)

    def embed(self, input_ids):
        return embed_stream(input_ids, self.token_embeddings.weight, self.scale)

    forward = embed


class FedolornLMHeadModel(LlamaLMHeadModel):
    """Shares the vocabulary handling and cache construction of the Llama head model; the head is the embedding itself."""

    def __init__(self, vocab_size: int, config: FedolornConfig, *, tp=None):
        nn.Module.__init__(self)
        if tp is not None and tp.size > 1:
            raise NotImplementedError("fedolorn has no tensor-parallel form")
        self.config = config
        self._vocab_size = vocab_size
        self.transformer = FedolornTransformer(config)
        self.embeddings = FedolornEmbedding(vocab_size, config)
        self.lm_head = None

    def activations(self, input_ids, attn_mask=None, *, pos_ids=None):
        return self.transformer(self.embeddings.embed(input_ids), attn_mask if attn_mask is not None else AttentionMask.causal(), pos_ids)

    def decode(self, input_ids, kv_cache, batch_info, pos_ids, logit_rows: Optional[torch.Tensor] = None):
        x = self.embeddings.embed(input_ids)
        h, kv_cache = self.transformer.decode(x, kv_cache, batch_info, pos_ids, logit_rows)
        return project(h, self.embeddings.token_embeddings.weight, out_dtype=torch.float32), kv_cache

    # -- checkpoint names ----------------------------------------------------------------------------------------
    def hf_tensor_names(self, name: str) -> Union[str, List[str]]:
        """Name of a parameter's tensor in a checkpoint; a list when the checkpoint keeps the slices of its first axis apart."""
        if name == "embeddings.token_embeddings.weight":
            return "embed"
        if name == "transformer.norm.weight":
            return "final.norm"
        i, rest = name[len("transformer.layers."):].split(".", 1)
        if rest.startswith("mlp.experts."):
            kind = rest.rsplit(".", 1)[1]
            return [f"l{i}.mlp.e{j}.{kind}" for j in range(self.config.layers[int(i)].num_experts)]
        fixed = {"input_layernorm.weight": "norm1", "post_attention_layernorm.weight": "norm2", "mlp.up_proj.weight": "mlp.up",
                 "mlp.down_proj.weight": "mlp.down", "mlp.router.weight": "mlp.router", "mlp.correction": "mlp.correction"}
        if rest in fixed:
            return f"l{i}.{fixed[rest]}"
        return f"l{i}.mix.{rest[len('self_attn.')]}"  # self_attn.{q,k,v,g,o}_proj.weight
