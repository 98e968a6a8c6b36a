"""Zadepel: a decoder-only model whose layers choose their token mixer: grouped-query attention with partial rotations, score
temperatures and mixed values; windowed latent attention; or a minimal gated recurrence.

Every layer describes itself (``ZadepelLayerConfig``): mixer, sizes and feed-forward may change from layer to layer.  With the residual
stream ``x`` in fp32 and ``N`` a plain RMS norm:

* ``x = E[token]``; per layer ``x += N1b(M(N1(x)))`` and, unless the layer has no feed-forward, ``x += N2b(F(N2(x)))``; logits are ``N(x)
  E^T``.
* ``M`` = attention: biased q, k, v; the first ``rotary_dim`` dimensions of a head rotate (halves paired); the scores of query head ``h``
  are multiplied by a learned number; in layers with ``value_mixing``, ``v <- (1 - m) v + m v_first`` with the values of the first such layer.
* ``M`` = latent attention: keys and values from a normed latent of ``kv_lora_rank`` and one rotated key part for all heads (neighbours
  paired); a query sees itself and the ``sliding_window - 1`` tokens before it.
* ``M`` = minGRU (``layers.recurrence.MinGru``).
* ``F``: ``W_down (gelu(W_gate h) * W_up h)`` with the tanh form of gelu.

Serving follows the other models' path (``decode`` over packed tokens).  Attention layers keep pages, recurrent layers a state per sequence
slot.  Between two sublayers one kernel norms the output, adds it to the stream and norms the sum (``ops.residual_stream``)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple, Type, Union

import torch
import torch.nn as nn
from torch.utils.checkpoint import checkpoint

from ..compat.hf_checkpoints import HFCheckpointConverter, HFCompatConfig
from ..layers.attention import (Attention, AttentionBackend, AttentionConfig, AttentionMask, MultiHeadLatentAttention,
                                MultiHeadLatentAttentionConfig)
from ..layers.normalization import LayerNormConfigBase, RmsNormConfig
from ..layers.recurrence import MinGru
from ..layers.rotary import DefaultRotaryEmbeddingsConfig
from ..nn import Embedding
from ..ops.residual_stream import add_norm_stream, embed_stream, project, rms_norm_stream
from ..utils.activation import ActivationFunctionEnum
from ..utils.remat import ScanCheckpointPolicy, should_recompute
from .llama import LlamaMlp, RecurrentLMHeadModel
from .lm_model import LmConfig

MIXERS = ("attention", "latent_attention", "mingru")


@dataclass(frozen=True)
class ZadepelLayerConfig:
    """Sizes of one layer.  ``intermediate_dim`` None: the layer has no feed-forward.  Which fields count depends on ``mixer``:

    * attention: ``num_heads``, ``num_kv_heads``, ``head_dim``, ``v_head_dim``, ``attention_scale``, ``rope_theta``, ``rotary_dim``,
      ``value_mixing``;
    * latent_attention: ``num_heads``, ``head_dim`` (the part without positions), ``rotary_dim`` (the rotated part), ``v_head_dim``,
      ``kv_lora_rank``, ``attention_scale``, ``rope_theta``, ``sliding_window`` (None: all earlier tokens);
    * mingru: ``width``."""

    mixer: str = "attention"
    num_heads: int = 32
    num_kv_heads: int = 8
    head_dim: int = 128
    v_head_dim: int = 128
    attention_scale: float = 128 ** -0.5
    rope_theta: float = 10000.0
    rotary_dim: int = 64
    value_mixing: bool = True
    kv_lora_rank: int = 512
    sliding_window: Optional[int] = None
    width: int = 4096
    intermediate_dim: Optional[int] = 14336

    def __post_init__(self):
        if self.mixer not in MIXERS:
            raise ValueError(f"unknown mixer {self.mixer!r}: one of {', '.join(MIXERS)}")
        if self.mixer == "attention":
            if self.num_heads % self.num_kv_heads != 0:
                raise ValueError(f"{self.num_heads} query heads cannot share {self.num_kv_heads} key/value heads")
            if not 0 < self.rotary_dim <= self.head_dim:
                raise ValueError(f"cannot rotate {self.rotary_dim} of {self.head_dim} dimensions")
        if self.mixer != "mingru" and self.rotary_dim % 2 != 0:
            raise ValueError("rotary_dim must be even")
        if self.sliding_window is not None and self.sliding_window <= 0:
            raise ValueError("sliding_window must be positive")


def _layer_from_checkpoint(entry: dict) -> ZadepelLayerConfig:
    kind, m, f = entry["type"], entry["mixer"], entry.get("mlp")
    if f is not None and f["kind"] != "dense":
        raise ValueError(f"unknown feed-forward kind {f['kind']!r}")
    kw = dict(mixer=kind, intermediate_dim=None if f is None else f["ff"])
    if kind == "attention":
        kw.update(num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], v_head_dim=m["vdim"], attention_scale=float(m["scale"]),
                  rope_theta=float(m["rot"]["base"]), rotary_dim=m["rot"]["dims"], value_mixing=bool(m.get("v_mix", False)))
    elif kind == "latent_attention":
        if m["rot"]["dims"] != m["rot_dim"]:
            raise ValueError(f"the rotated part has {m['rot_dim']} dimensions but {m['rot']['dims']} of them are to rotate")
        mask = m.get("mask")
        kw.update(num_heads=m["heads"], head_dim=m["dim"], v_head_dim=m["vdim"], kv_lora_rank=m["kv_rank"], attention_scale=float(m["scale"]),
                  rope_theta=float(m["rot"]["base"]), rotary_dim=m["rot_dim"], sliding_window=None if mask is None else mask["size"])
    elif kind == "mingru":
        kw.update(width=m["width"])
    return ZadepelLayerConfig(**kw)


def _layer_to_checkpoint(c: ZadepelLayerConfig) -> dict:
    rot = dict(base=c.rope_theta, dims=c.rotary_dim)
    if c.mixer == "attention":
        m = dict(heads=c.num_heads, kv_heads=c.num_kv_heads, dim=c.head_dim, vdim=c.v_head_dim, scale=c.attention_scale, rot=rot, v_mix=c.value_mixing)
    elif c.mixer == "latent_attention":
        m = dict(heads=c.num_heads, dim=c.head_dim, vdim=c.v_head_dim, kv_rank=c.kv_lora_rank, scale=c.attention_scale, rot=rot, rot_dim=c.rotary_dim)
        if c.sliding_window is not None:
            m["mask"] = {"size": c.sliding_window}
    else:
        m = dict(width=c.width)
    return dict(type=c.mixer, mixer=m, mlp=None if c.intermediate_dim is None else dict(kind="dense", ff=c.intermediate_dim))


@LmConfig.register_subclass("zadepel")
@dataclass(frozen=True)
class ZadepelConfig(HFCompatConfig):
    seq_len: int = 8192
    hidden_dim: int = 4096
    layer_norm_epsilon: float = 1e-6
    layers: Tuple[ZadepelLayerConfig, ...] = (ZadepelLayerConfig(),)
    initializer_range: float = 0.02
    upcast_attn: bool = False
    attn_backend: Optional[AttentionBackend] = None
    gradient_checkpointing: Union[bool, ScanCheckpointPolicy, str] = True
    reference_checkpoint: Optional[str] = None
    tokenizer: Optional[str] = None
    cross_entropy_block_size: Optional[int] = None

    hf_architecture = "Zadepel"
    hf_vocab_key = "vocab"
    tie_word_embeddings = True

    def __post_init__(self):
        layers = tuple(ZadepelLayerConfig(**l) if isinstance(l, dict) else l for l in self.layers)
        object.__setattr__(self, "layers", layers)
        if not layers:
            raise ValueError("a model has at least one layer")
        if len({(l.num_kv_heads, l.v_head_dim) for l in layers if l.mixer == "attention" and l.value_mixing}) > 1:
            raise ValueError("layers that mix values must have the same key/value heads and value size")

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def model_type(self) -> Type["ZadepelLMHeadModel"]:
        return ZadepelLMHeadModel

    def hf_checkpoint_converter(self, ref_checkpoint: Optional[str] = None) -> HFCheckpointConverter:
        return HFCheckpointConverter(self.__class__, reference_checkpoint=ref_checkpoint or self.reference_checkpoint,
                                     tokenizer=ref_checkpoint if self.tokenizer is None else self.tokenizer)

    @classmethod
    def from_hf_config(cls, hf_config) -> "ZadepelConfig":
        c = hf_config if isinstance(hf_config, dict) else vars(hf_config)
        return cls(hidden_dim=c["width"], layer_norm_epsilon=float(c["norm"]["eps"]), layers=tuple(_layer_from_checkpoint(l) for l in c["layers"]))

    def to_hf_config(self, vocab_size: int, config_overrides: Optional[Dict] = None) -> dict:
        cfg = dict(architecture=self.hf_architecture, vocab=vocab_size, width=self.hidden_dim, norm={"eps": self.layer_norm_epsilon},
                   layers=[_layer_to_checkpoint(l) for l in self.layers])
        cfg.update(config_overrides or {})
        return cfg

    @property
    def norm_config(self) -> LayerNormConfigBase:
        return RmsNormConfig(eps=self.layer_norm_epsilon, use_weight=True, use_bias=False)

    def mk_LayerNorm(self, dim: int):
        return self.norm_config.build(dim)

    def build_mixer(self, l: ZadepelLayerConfig) -> nn.Module:
        std = self.initializer_range
        if l.mixer == "mingru":
            return MinGru(self.hidden_dim, l.width, init_std=std)
        if l.mixer == "latent_attention":
            rope = DefaultRotaryEmbeddingsConfig(theta=l.rope_theta, interleaved=True)
            return MultiHeadLatentAttention(MultiHeadLatentAttentionConfig(
                hidden_dim=self.hidden_dim, num_heads=l.num_heads, kv_lora_rank=l.kv_lora_rank, qk_rope_head_dim=l.rotary_dim, qk_nope_head_dim=l.head_dim,
                v_head_dim=l.v_head_dim, upcast_attn=self.upcast_attn, attn_backend=self.attn_backend, rope=rope, scaling_factor=l.attention_scale,
                norm_eps=self.layer_norm_epsilon, sliding_window=l.sliding_window), init_std=std)
        rope = DefaultRotaryEmbeddingsConfig(theta=l.rope_theta, rotary_dim=l.rotary_dim)
        return Attention(AttentionConfig(
            hidden_dim=self.hidden_dim, num_heads=l.num_heads, num_kv_heads=l.num_kv_heads, head_dim=l.head_dim, v_head_dim=l.v_head_dim, use_bias=True,
            use_output_bias=False, upcast_attn=self.upcast_attn, attn_backend=self.attn_backend, rope=rope, scaling_factor=l.attention_scale,
            head_temperature=True, value_mixing=l.value_mixing), init_std=std)

    def _products(self, l: ZadepelLayerConfig) -> int:
        """Weights of a layer's matrix products."""
        e, H = self.hidden_dim, l.num_heads
        n = 0 if l.intermediate_dim is None else 3 * e * l.intermediate_dim
        if l.mixer == "mingru":
            return n + 4 * e * l.width
        if l.mixer == "latent_attention":
            r = l.kv_lora_rank
            return n + e * (H * (l.head_dim + l.rotary_dim + l.v_head_dim) + r + l.rotary_dim) + r * H * (l.head_dim + l.v_head_dim)
        return n + e * (H + l.num_kv_heads) * (l.head_dim + l.v_head_dim)

    def flops_per_token(self, vocab_size: int) -> float:
        attn = 0.0
        for l in self.layers:
            if l.mixer == "attention":
                attn += 2 * l.num_heads * (l.head_dim + l.v_head_dim) * self.seq_len
            elif l.mixer == "latent_attention":
                attn += 2 * l.num_heads * (l.head_dim + l.rotary_dim + l.v_head_dim) * min(l.sliding_window or self.seq_len, self.seq_len)
            else:
                attn += 8 * l.width
        return 2.0 * (sum(self._products(l) for l in self.layers) + vocab_size * self.hidden_dim) + attn

    def total_trainable_params(self, vocab_size: int) -> int:
        e = self.hidden_dim
        n = e + vocab_size * e
        for l in self.layers:
            n += self._products(l) + (2 * e if l.intermediate_dim is None else 4 * e)
            if l.mixer == "attention":
                n += l.num_heads * (l.head_dim + 1) + l.num_kv_heads * (l.head_dim + l.v_head_dim) + int(l.value_mixing)
            else:
                n += l.kv_lora_rank if l.mixer == "latent_attention" else 2 * l.width
        return n


class ZadepelDecoderLayer(nn.Module):
    """``x`` is the fp32 stream; the norms before a sublayer hand it the compute dtype, the norms after it work on its fp32 output."""

    def __init__(self, config: ZadepelConfig, layer: ZadepelLayerConfig):
        super().__init__()
        self.kind = layer.mixer
        self.mixer = config.build_mixer(layer)
        self.input_layernorm = config.mk_LayerNorm(config.hidden_dim)
        self.post_mixer_layernorm = config.mk_LayerNorm(config.hidden_dim)
        self.mlp = None
        if layer.intermediate_dim is not None:
            self.pre_mlp_layernorm = config.mk_LayerNorm(config.hidden_dim)
            self.post_mlp_layernorm = config.mk_LayerNorm(config.hidden_dim)
            self.mlp = LlamaMlp(config.hidden_dim, layer.intermediate_dim, ActivationFunctionEnum.gelu_new, init_std=config.initializer_range)

    @staticmethod
    def _normed_in_fp32(norm, y: torch.Tensor) -> torch.Tensor:
        return rms_norm_stream(y.float(), norm.weight, norm.eps, out_dtype=torch.float32)

    def forward(self, x, mask=None, pos_ids=None, v_first=None):
        h = self.input_layernorm.from_stream(x)
        if self.kind == "attention":
            y, v_first = self.mixer.forward_mixing_values(h, mask, pos_ids, v_first)
        else:
            y = self.mixer(h, mask, pos_ids)
        x = x + self._normed_in_fp32(self.post_mixer_layernorm, y)
        if self.mlp is not None:
            x = x + self._normed_in_fp32(self.post_mlp_layernorm, self.mlp(self.pre_mlp_layernorm.from_stream(x)))
        return x, v_first

    def mix(self, h, cache, batch_info, pos_ids, v_first):
        """The mixer over packed rows of a serving step: ``(output in fp32, v_first)``."""
        if self.kind == "attention":
            return self.mixer.paged_decode_mixing_values(h, cache, batch_info, pos_ids, v_first)
        return self.mixer.paged_decode(h, cache, batch_info, pos_ids), v_first


class ZadepelTransformer(nn.Module):
    def __init__(self, config: ZadepelConfig):
        super().__init__()
        self.config = config
        self.layers = nn.ModuleList([ZadepelDecoderLayer(config, l) for l in config.layers])
        self.norm = config.mk_LayerNorm(config.hidden_dim)

    def forward(self, x, mask=None, pos_ids=None):
        remat = should_recompute(self.config.gradient_checkpointing) and torch.is_grad_enabled() and self.training
        v_first = None
        for layer in self.layers:
            x, v_first = checkpoint(layer, x, mask, pos_ids, v_first, use_reentrant=False) if remat else layer(x, mask, pos_ids, v_first)
        return self.norm.from_stream(x)

    def decode(self, x, caches, batch_info, pos_ids, logit_rows=None):
        eps, n = self.config.layer_norm_epsilon, len(self.layers)
        h = self.layers[0].input_layernorm.from_stream(x)
        v_first = None
        for i, (layer, cache) in enumerate(zip(self.layers, caches)):
            last = i + 1 == n
            after = self.norm if last else self.layers[i + 1].input_layernorm  # what the sum after this layer's last sublayer is normed by
            rows = logit_rows if last else None
            y, v_first = layer.mix(h, cache, batch_info, pos_ids, v_first)
            if layer.mlp is None:
                h = add_norm_stream(x, y, layer.post_mixer_layernorm.weight, after.weight, eps, rows=rows)
                continue
            h = add_norm_stream(x, y, layer.post_mixer_layernorm.weight, layer.pre_mlp_layernorm.weight, eps)
            h = add_norm_stream(x, layer.mlp.forward_fp32(h), layer.post_mlp_layernorm.weight, after.weight, eps, rows=rows)
        return h, caches

    def initial_cache(self, max_pages: int, page_size: int, max_seqs: int, *, dtype=torch.bfloat16, device=None):
        return [l.mixer.empty_state(max_seqs, device=device) if l.kind == "mingru" else
                l.mixer.empty_page_cache(max_pages, page_size, dtype=dtype, device=device) for l in self.layers]


class ZadepelEmbedding(nn.Module):
    def __init__(self, vocab_size: int, config: ZadepelConfig):
        super().__init__()
        self.token_embeddings = Embedding(vocab_size, config.hidden_dim, init_std=config.initializer_range)

    def embed(self, input_ids):
        return embed_stream(input_ids, self.token_embeddings.weight, 1.0)

    forward = embed


class ZadepelLMHeadModel(RecurrentLMHeadModel):
    """Shares the vocabulary handling of the Llama head model; the head is the embedding itself."""

    def __init__(self, vocab_size: int, config: ZadepelConfig, *, tp=None):
        nn.Module.__init__(self)
        if tp is not None and tp.size > 1:
            raise NotImplementedError("zadepel has no tensor-parallel form")
        self.config = config
        self._vocab_size = vocab_size
        self.transformer = ZadepelTransformer(config)
        self.embeddings = ZadepelEmbedding(vocab_size, config)
        self.lm_head = None

    def activations(self, input_ids, attn_mask=None, *, pos_ids=None):
        return self.transformer(self.embeddings.embed(input_ids), attn_mask if attn_mask is not None else AttentionMask.causal(), pos_ids)

    def decode(self, input_ids, kv_cache, batch_info, pos_ids, logit_rows: Optional[torch.Tensor] = None):
        x = self.embeddings.embed(input_ids)
        h, kv_cache = self.transformer.decode(x, kv_cache, batch_info, pos_ids, logit_rows)
        return project(h, self.embeddings.token_embeddings.weight, out_dtype=torch.float32), kv_cache

    # -- checkpoint names ----------------------------------------------------------------------------------------
    def hf_tensor_parts(self, name: str, t: torch.Tensor) -> List[Tuple[str, torch.Tensor, Tuple[int, ...]]]:
        """``(checkpoint tensor, view of t, its shape in the checkpoint)`` of a parameter's value ``t``."""
        if name == "embeddings.token_embeddings.weight":
            return [("embed", t, t.shape)]
        if name == "transformer.norm.weight":
            return [("final.norm", t, t.shape)]
        i, rest = name[len("transformer.layers."):].split(".", 1)
        if rest == "mixer.kv_b_proj.weight":
            mixer = self.transformer.layers[int(i)].mixer
            return [(f"l{i}.mix.{n}", v, (v.shape[0] * v.shape[1], v.shape[2])) for n, v in zip(("uk", "uv"), mixer.up_projections(t))]
        fixed = {"input_layernorm.weight": "norm1", "post_mixer_layernorm.weight": "norm1b", "pre_mlp_layernorm.weight": "norm2",
                 "post_mlp_layernorm.weight": "norm2b", "mlp.gate_proj.weight": "mlp.gate", "mlp.up_proj.weight": "mlp.up",
                 "mlp.down_proj.weight": "mlp.down", "mixer.temperature": "mix.temp", "mixer.value_mix": "mix.vmix", "mixer.kv_a_proj.weight": "mix.dkv",
                 "mixer.kv_a_norm.weight": "mix.dkv.norm"}
        if rest in fixed:
            return [(f"l{i}.{fixed[rest]}", t, t.shape)]
        proj, kind = rest[len("mixer."):].rsplit(".", 1)  # mixer.{q,k,v,z,x,g,o}_proj.{weight,bias}
        return [(f"l{i}.mix.{proj[:-len('_proj')]}" + (".b" if kind == "bias" else ""), t, t.shape)]
