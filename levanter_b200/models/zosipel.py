"""Zosipel: a decoder-only model of differential-attention and latent-attention layers with mixture feed-forwards, a range of which runs
several times over.

Every layer describes itself (``ZosipelLayerConfig``): mixer, sizes and feed-forward may change from layer to layer.  With the residual
stream ``x`` in fp32 and ``N`` an RMS norm with weight ``1 + w``:

* ``x = E[token]``; per layer ``x += M(N1(x))`` and, unless the layer has no feed-forward, ``x += F(N2(x))``; logits are ``W N(x)``.
* Layers ``loop_start .. loop_stop - 1`` run ``loop_times`` times in a row with the same weights; before pass ``t`` a learned vector
  ``step[t]`` joins the stream.  Every pass has pages of its own.
* ``M`` = attention: two score maps per head over the same values, with biased q, k, v, a (YaRN) rotation of the first dimensions, soft-capped
  scores and a sliding window; the maps' difference is normed (``ops.map_difference``) and gated by one number per head.
* ``M`` = latent attention without positions, with a learned sink per head in the softmax denominator.
* ``F``: ``layers.experts.GroupedSoftmaxMoe``.

Serving follows the other models' path (``decode`` over packed tokens and a paged cache)."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple, Type, Union

import torch
import torch.nn as nn
from torch.utils.checkpoint import checkpoint

from ..compat.hf_checkpoints import HFCheckpointConverter, HFCompatConfig
from ..layers.attention import (Attention, AttentionBackend, AttentionConfig, AttentionMask, MultiHeadLatentAttention,
                                MultiHeadLatentAttentionConfig)
from ..layers.experts import GroupedSoftmaxMoe
from ..layers.normalization import LayerNormConfigBase
from ..layers.rotary import DefaultRotaryEmbeddingsConfig, RotaryEmbeddingsConfig, rope_from_entry, rope_to_entry
from ..nn import Embedding, Linear
from ..ops.residual_stream import embed_stream, project
from ..utils.remat import ScanCheckpointPolicy, should_recompute
from .gemma import GemmaNormConfig
from .llama import LlamaLMHeadModel
from .lm_model import LmConfig

MIXERS = ("attention", "latent_attention")


@dataclass(frozen=True)
class ZosipelLayerConfig:
    """Sizes of one layer.  Which fields count depends on ``mixer``:

    * attention: ``num_heads``, ``num_kv_heads``, ``head_dim`` (of each of the two maps), ``v_head_dim``, ``attention_scale``, ``rope``,
      ``difference`` (the constant part of the second map's weight), ``soft_cap`` and ``sliding_window`` (None: none);
    * latent_attention: ``num_heads``, ``head_dim``, ``v_head_dim``, ``kv_lora_rank``, ``attention_scale``.

    ``intermediate_dim`` is an expert's; None: the layer has no feed-forward.  ``shared_intermediate_dim`` None: no shared expert."""

    mixer: str = "attention"
    num_heads: int = 16
    num_kv_heads: int = 4
    head_dim: int = 64
    v_head_dim: int = 128
    attention_scale: float = 64 ** -0.5
    rope: Optional[RotaryEmbeddingsConfig] = field(default_factory=DefaultRotaryEmbeddingsConfig)
    difference: float = 0.8
    soft_cap: Optional[float] = None
    sliding_window: Optional[int] = None
    kv_lora_rank: int = 512
    intermediate_dim: Optional[int] = 1024
    num_experts: int = 64
    num_experts_per_tok: int = 8
    expert_groups: int = 1
    expert_groups_kept: int = 1
    shared_intermediate_dim: Optional[int] = None

    def __post_init__(self):
        if self.mixer not in MIXERS:
            raise ValueError(f"unknown mixer {self.mixer!r}: one of {', '.join(MIXERS)}")
        if self.mixer == "attention":
            if self.num_heads % self.num_kv_heads != 0:
                raise ValueError(f"{self.num_heads} query heads cannot share {self.num_kv_heads} key/value heads")
            if self.rope is not None:
                self.rope.build(self.head_dim)  # rejects what cannot be rotated
        for name in ("soft_cap", "sliding_window"):
            if getattr(self, name) is not None and getattr(self, name) <= 0:
                raise ValueError(f"{name} must be positive")
        if self.intermediate_dim is not None:
            if self.num_experts <= 0 or self.num_experts % self.expert_groups != 0:
                raise ValueError(f"{self.num_experts} experts do not form {self.expert_groups} equal groups")
            if not 0 < self.expert_groups_kept <= self.expert_groups:
                raise ValueError(f"cannot keep {self.expert_groups_kept} of {self.expert_groups} expert groups")
            if not 0 < self.num_experts_per_tok <= self.expert_groups_kept * (self.num_experts // self.expert_groups):
                raise ValueError(f"{self.num_experts_per_tok} experts per token do not fit the kept groups")


def _layer_from_checkpoint(entry: dict) -> ZosipelLayerConfig:
    kind, m, f = entry["type"], entry["mixer"], entry.get("mlp")
    kw = dict(mixer=kind, num_heads=m["heads"], head_dim=m["dim"], v_head_dim=m["vdim"], attention_scale=float(m["scale"]), intermediate_dim=None)
    if kind == "attention":
        mask, cap = m.get("mask"), m.get("softcap")
        kw.update(num_kv_heads=m["kv_heads"], rope=rope_from_entry(m.get("rot")), difference=float(m["diff"]),
                  soft_cap=None if cap is None else float(cap), sliding_window=None if mask is None else mask["size"])
    elif kind == "latent_attention":
        kw.update(kv_lora_rank=m["kv_rank"], rope=None)
    if f is not None:
        if f["kind"] != "moe":
            raise ValueError(f"unknown feed-forward kind {f['kind']!r}")
        r, shared = f["router"], f.get("shared")
        g = r.get("groups") or {"count": 1, "keep": 1}
        kw.update(intermediate_dim=f["expert"]["ff"], num_experts=r["experts"], num_experts_per_tok=r["top"], expert_groups=g["count"],
                  expert_groups_kept=g["keep"], shared_intermediate_dim=None if shared is None else shared["ff"])
    return ZosipelLayerConfig(**kw)


def _layer_to_checkpoint(c: ZosipelLayerConfig) -> dict:
    m = dict(heads=c.num_heads, dim=c.head_dim, vdim=c.v_head_dim, scale=c.attention_scale)
    if c.mixer == "attention":
        m.update(kv_heads=c.num_kv_heads, diff=c.difference)
        if c.rope is not None:
            m["rot"] = rope_to_entry(c.rope, c.head_dim)
        if c.soft_cap is not None:
            m["softcap"] = c.soft_cap
        if c.sliding_window is not None:
            m["mask"] = {"size": c.sliding_window}
    else:
        m.update(kv_rank=c.kv_lora_rank)
    mlp = None
    if c.intermediate_dim is not None:
        mlp = dict(kind="moe", expert={"ff": c.intermediate_dim},
                   router=dict(experts=c.num_experts, top=c.num_experts_per_tok, groups={"count": c.expert_groups, "keep": c.expert_groups_kept}))
        if c.shared_intermediate_dim is not None:
            mlp["shared"] = {"ff": c.shared_intermediate_dim}
    return dict(type=c.mixer, mixer=m, mlp=mlp)


@LmConfig.register_subclass("zosipel")
@dataclass(frozen=True)
class ZosipelConfig(HFCompatConfig):
    """``loop_times`` 0: every layer runs once and there are no pass vectors."""

    seq_len: int = 8192
    hidden_dim: int = 2048
    layer_norm_epsilon: float = 1e-6
    layers: Tuple[ZosipelLayerConfig, ...] = (ZosipelLayerConfig(),)
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 0
    initializer_range: float = 0.02
    upcast_attn: bool = False
    attn_backend: Optional[AttentionBackend] = None
    gradient_checkpointing: Union[bool, ScanCheckpointPolicy, str] = True
    reference_checkpoint: Optional[str] = None
    tokenizer: Optional[str] = None
    cross_entropy_block_size: Optional[int] = None

    hf_architecture = "Zosipel"
    hf_vocab_key = "vocab"
    tie_word_embeddings = False

    def __post_init__(self):
        layers = tuple(ZosipelLayerConfig(**l) if isinstance(l, dict) else l for l in self.layers)
        object.__setattr__(self, "layers", layers)
        if not layers:
            raise ValueError("a model has at least one layer")
        if self.loop_times < 0 or (self.loop_times > 0 and not 0 <= self.loop_start < self.loop_stop <= len(layers)):
            raise ValueError(f"layers {self.loop_start} .. {self.loop_stop - 1} of {len(layers)} cannot run {self.loop_times} times")

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def layer_runs(self) -> List[Tuple[int, Optional[int]]]:
        """The layers in the order they run: ``(layer, number of the pass that it begins, or None)``."""
        n = len(self.layers)
        if self.loop_times == 0:
            return [(i, None) for i in range(n)]
        runs: List[Tuple[int, Optional[int]]] = [(i, None) for i in range(self.loop_start)]
        for t in range(self.loop_times):
            runs += [(i, t if i == self.loop_start else None) for i in range(self.loop_start, self.loop_stop)]
        return runs + [(i, None) for i in range(self.loop_stop, n)]

    @property
    def model_type(self) -> Type["ZosipelLMHeadModel"]:
        return ZosipelLMHeadModel

    def hf_checkpoint_converter(self, ref_checkpoint: Optional[str] = None) -> HFCheckpointConverter:
        return HFCheckpointConverter(self.__class__, reference_checkpoint=ref_checkpoint or self.reference_checkpoint,
                                     tokenizer=ref_checkpoint if self.tokenizer is None else self.tokenizer)

    @classmethod
    def from_hf_config(cls, hf_config) -> "ZosipelConfig":
        c = hf_config if isinstance(hf_config, dict) else vars(hf_config)
        loop = c.get("loop")
        kw = {} if loop is None else dict(loop_start=loop["start"], loop_stop=loop["stop"], loop_times=loop["times"])
        return cls(hidden_dim=c["width"], layer_norm_epsilon=float(c["norm"]["eps"]), layers=tuple(_layer_from_checkpoint(l) for l in c["layers"]), **kw)

    def to_hf_config(self, vocab_size: int, config_overrides: Optional[Dict] = None) -> dict:
        cfg = dict(architecture=self.hf_architecture, vocab=vocab_size, width=self.hidden_dim, norm={"eps": self.layer_norm_epsilon},
                   layers=[_layer_to_checkpoint(l) for l in self.layers])
        if self.loop_times > 0:
            cfg["loop"] = dict(start=self.loop_start, stop=self.loop_stop, times=self.loop_times)
        cfg.update(config_overrides or {})
        return cfg

    @property
    def norm_config(self) -> LayerNormConfigBase:
        return GemmaNormConfig(eps=self.layer_norm_epsilon, use_weight=True, use_bias=False)

    def mk_LayerNorm(self, dim: int):
        return self.norm_config.build(dim)

    def build_mixer(self, l: ZosipelLayerConfig) -> nn.Module:
        std = self.initializer_range
        if l.mixer == "latent_attention":
            return MultiHeadLatentAttention(MultiHeadLatentAttentionConfig(
                hidden_dim=self.hidden_dim, num_heads=l.num_heads, kv_lora_rank=l.kv_lora_rank, qk_rope_head_dim=0, qk_nope_head_dim=l.head_dim,
                v_head_dim=l.v_head_dim, upcast_attn=self.upcast_attn, attn_backend=self.attn_backend, scaling_factor=l.attention_scale,
                norm_eps=self.layer_norm_epsilon, sink=True), init_std=std)
        return Attention(AttentionConfig(
            hidden_dim=self.hidden_dim, num_heads=l.num_heads, num_kv_heads=l.num_kv_heads, head_dim=l.head_dim, v_head_dim=l.v_head_dim, use_bias=True,
            use_output_bias=False, upcast_attn=self.upcast_attn, attn_backend=self.attn_backend, rope=l.rope, scaling_factor=l.attention_scale,
            logits_soft_cap=l.soft_cap, sliding_window=l.sliding_window, head_gate=True, differential=l.difference,
            norm_eps=self.layer_norm_epsilon), init_std=std)

    def _products(self, l: ZosipelLayerConfig, active: bool) -> int:
        """Weights of a layer's matrix products (``active``: of those that a token uses)."""
        e, H = self.hidden_dim, l.num_heads
        if l.mixer == "latent_attention":
            r = l.kv_lora_rank
            n = e * (H * (l.head_dim + l.v_head_dim) + r) + r * H * (l.head_dim + l.v_head_dim)
        else:
            n = e * (2 * H * l.head_dim + H * l.v_head_dim + H + l.num_kv_heads * (2 * l.head_dim + l.v_head_dim))
        if l.intermediate_dim is not None:
            n += e * l.num_experts + 3 * e * l.intermediate_dim * (l.num_experts_per_tok if active else l.num_experts)
            if l.shared_intermediate_dim is not None:
                n += 3 * e * l.shared_intermediate_dim + e
        return n

    def flops_per_token(self, vocab_size: int) -> float:
        flops = 2.0 * vocab_size * self.hidden_dim
        for i, _ in self.layer_runs():
            l = self.layers[i]
            keys = min(l.sliding_window or self.seq_len, self.seq_len) if l.mixer == "attention" else self.seq_len
            flops += 2.0 * self._products(l, True) + 2 * (2 if l.mixer == "attention" else 1) * l.num_heads * (l.head_dim + l.v_head_dim) * keys
        return flops

    def total_trainable_params(self, vocab_size: int) -> int:
        e = self.hidden_dim
        n = e + 2 * vocab_size * e + self.loop_times * e
        for l in self.layers:
            n += self._products(l, False) + (e if l.intermediate_dim is None else 2 * e)
            if l.mixer == "attention":
                n += 2 * l.num_heads * l.head_dim + l.num_kv_heads * (2 * l.head_dim + l.v_head_dim) + 4 * l.head_dim
            else:
                n += l.kv_lora_rank + l.num_heads
        return n


class ZosipelDecoderLayer(nn.Module):
    """``x`` is the fp32 stream; the norms hand the compute dtype to the mixer and the feed-forward.  ``add``: a vector that joins the
    stream first."""

    def __init__(self, config: ZosipelConfig, layer: ZosipelLayerConfig):
        super().__init__()
        self.mixer = config.build_mixer(layer)
        self.input_layernorm = config.mk_LayerNorm(config.hidden_dim)
        self.mlp = None
        if layer.intermediate_dim is not None:
            self.post_attention_layernorm = config.mk_LayerNorm(config.hidden_dim)
            self.mlp = GroupedSoftmaxMoe(config.hidden_dim, layer.intermediate_dim, layer.num_experts, layer.num_experts_per_tok,
                                         groups=layer.expert_groups, keep=layer.expert_groups_kept,
                                         shared_intermediate=layer.shared_intermediate_dim, init_std=config.initializer_range)

    def _feed_forward(self, x, batch_info=None):
        if self.mlp is None:
            return x
        return self.mlp.add_to_stream(x, self.post_attention_layernorm.from_stream(x), batch_info)

    def forward(self, x, mask=None, pos_ids=None, add=None):
        if add is not None:
            x = x + add.float()
        x = x + self.mixer(self.input_layernorm.from_stream(x), mask, pos_ids).float()
        return self._feed_forward(x)

    def decode(self, x, kv_cache, batch_info, pos_ids, add=None):
        h = self.input_layernorm.from_stream(x, add=add)
        x, kv_cache = self.mixer.paged_decode_stream(h, kv_cache, batch_info, pos_ids, x)
        return self._feed_forward(x, batch_info), kv_cache


class ZosipelTransformer(nn.Module):
    def __init__(self, config: ZosipelConfig):
        super().__init__()
        self.config = config
        self.layers = nn.ModuleList([ZosipelDecoderLayer(config, l) for l in config.layers])
        self.runs = config.layer_runs()
        if config.loop_times > 0:
            self.loop_step = nn.Parameter(torch.randn(config.loop_times, config.hidden_dim) * config.initializer_range)
            self.loop_step.lev_shape = (config.loop_times, config.hidden_dim)
        self.norm = config.mk_LayerNorm(config.hidden_dim)

    def _step(self, t: Optional[int]) -> Optional[torch.Tensor]:
        return None if t is None else self.loop_step[t]

    def forward(self, x, mask=None, pos_ids=None):
        remat = should_recompute(self.config.gradient_checkpointing) and torch.is_grad_enabled() and self.training
        for i, t in self.runs:
            args = (x, mask, pos_ids, self._step(t))
            x = checkpoint(self.layers[i], *args, use_reentrant=False) if remat else self.layers[i](*args)
        return self.norm.from_stream(x)

    def decode(self, x, caches, batch_info, pos_ids, logit_rows=None):
        """``caches``: one per layer run."""
        new = []
        for (i, t), c in zip(self.runs, caches):
            x, c = self.layers[i].decode(x, c, batch_info, pos_ids, self._step(t))
            new.append(c)
        return self.norm.from_stream(x, rows=logit_rows), new

    def initial_cache(self, max_pages: int, page_size: int, *, dtype=torch.bfloat16, device=None):
        return [self.layers[i].mixer.empty_page_cache(max_pages, page_size, dtype=dtype, device=device) for i, _ in self.runs]


class ZosipelEmbedding(nn.Module):
    def __init__(self, vocab_size: int, config: ZosipelConfig):
        super().__init__()
        self.token_embeddings = Embedding(vocab_size, config.hidden_dim, init_std=config.initializer_range)

    def embed(self, input_ids):
        return embed_stream(input_ids, self.token_embeddings.weight, 1.0)

    forward = embed


class ZosipelLMHeadModel(LlamaLMHeadModel):
    """Shares the vocabulary handling and cache construction of the Llama head model."""

    def __init__(self, vocab_size: int, config: ZosipelConfig, *, tp=None):
        nn.Module.__init__(self)
        if tp is not None and tp.size > 1:
            raise NotImplementedError("zosipel has no tensor-parallel form")
        self.config = config
        self._vocab_size = vocab_size
        self.transformer = ZosipelTransformer(config)
        self.embeddings = ZosipelEmbedding(vocab_size, config)
        self.lm_head = Linear(config.hidden_dim, vocab_size, init_std=config.initializer_range)

    def activations(self, input_ids, attn_mask=None, *, pos_ids=None):
        return self.transformer(self.embeddings.embed(input_ids), attn_mask if attn_mask is not None else AttentionMask.causal(), pos_ids)

    def decode(self, input_ids, kv_cache, batch_info, pos_ids, logit_rows: Optional[torch.Tensor] = None):
        x = self.embeddings.embed(input_ids)
        h, kv_cache = self.transformer.decode(x, kv_cache, batch_info, pos_ids, logit_rows)
        return project(h, self.get_lm_head(), out_dtype=torch.float32), kv_cache

    # -- checkpoint names ----------------------------------------------------------------------------------------
    def hf_tensor_parts(self, name: str, t: torch.Tensor) -> List[Tuple[str, torch.Tensor, Tuple[int, ...]]]:
        """``(checkpoint tensor, view of t, its shape in the checkpoint)`` of a parameter's value ``t``."""
        top = {"embeddings.token_embeddings.weight": "embed", "lm_head.weight": "head", "transformer.norm.weight": "final.norm",
               "transformer.loop_step": "loop.step"}
        if name in top:
            return [(top[name], t, t.shape)]
        i, rest = name[len("transformer.layers."):].split(".", 1)
        pre = f"l{i}."
        if rest == "mixer.kv_b_proj.weight":
            mixer = self.transformer.layers[int(i)].mixer
            return [(f"{pre}mix.{n}", v, (v.shape[0] * v.shape[1], v.shape[2])) for n, v in zip(("uk", "uv"), mixer.up_projections(t))]
        if rest == "mlp.experts.gate_up":
            ff = t.shape[1] // 2
            return [(f"{pre}mlp.e{j}.{n}", v, v.shape) for j in range(t.shape[0]) for n, v in (("gate", t[j, :ff]), ("up", t[j, ff:]))]
        if rest == "mlp.experts.down":
            return [(f"{pre}mlp.e{j}.down", t[j], t.shape[1:]) for j in range(t.shape[0])]
        fixed = {"input_layernorm.weight": "norm1", "post_attention_layernorm.weight": "norm2", "mixer.kv_a_proj.weight": "mix.dkv",
                 "mixer.kv_a_norm.weight": "mix.dkv.norm", "mixer.sinks": "mix.sink", "mlp.router.weight": "mlp.router",
                 "mlp.shared_gate.weight": "mlp.shared.sg"}
        if rest in fixed:
            return [(pre + fixed[rest], t, t.shape)]
        if rest.startswith("mixer.lambda_"):
            return [(f"{pre}mix.l{rest[len('mixer.lambda_'):]}", t, t.shape)]
        owner, proj, kind = rest.rsplit(".", 2)  # mixer.{q,k,v,g,o}_proj.{weight,bias}, mlp.shared.{gate,up,down}_proj.weight
        owner = {"mixer": "mix", "mlp.shared": "mlp.shared"}[owner]
        return [(f"{pre}{owner}.{proj[:-len('_proj')]}" + (".b" if kind == "bias" else ""), t, t.shape)]
