"""Mumizen: a decoder-only model whose layers mix tokens by linear attention with fixed decays (two forms) or by latent attention, and whose
blocks start from a learned average over the results of all layers so far.

Every layer describes itself (``MumizenLayerConfig``): mixer, sizes and feed-forward may change from layer to layer.  With ``N`` an RMS norm
in groups and everything that joins the residual stream in fp32:

* ``X_0 = E[token]``; layer ``i`` starts from ``x`` (``X_0`` for the first): ``x += M(shift(N1(x)))`` and, unless the layer has no feed-forward, ``x +=
  F(N2(x))``; its result is ``X_{i+1} = x``, and ``sum_j a_i[j] X_j`` over ``j <= i + 1`` is what the next layer, or the final norm, starts from.
  Logits are ``W N(x)``.
* ``shift``: ``h + (h' - h) * mu`` with the previous token's ``h'``.
* ``M`` = lightning or retention: ``layers.recurrence.LinearAttention``.
* ``M`` = latent attention: queries through a latent of their own, a (YaRN) rotated part beside the unrotated one, an output gate; a layer
  may read the latents and rotated key parts that an earlier layer keeps (``kv_from``).
* ``F``: a gated feed-forward with bounded inputs (``ops.glu.ClampedGlu``), or ``layers.experts.GroupedSoftmaxMoe`` of such.

Serving follows the other models' path (``decode`` over packed tokens).  Latent attention keeps pages, linear attention a matrix state and
every layer the last normed row per sequence slot.  The results of the layers are the planes of one tensor; a block's projections
accumulate into its plane, and one kernel forms the average, the norm and the shift (``ops.depth_stream``)."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple, Type, Union

import torch
import torch.nn as nn
from torch.utils.checkpoint import checkpoint

from ..compat.hf_checkpoints import HFCheckpointConverter, HFCompatConfig
from ..layers.attention import AttentionBackend, AttentionMask, MultiHeadLatentAttention, MultiHeadLatentAttentionConfig
from ..layers.experts import GroupedSoftmaxMoe
from ..layers.normalization import GroupedRmsNormConfig, LayerNormConfigBase
from ..layers.recurrence import LinearAttention, LinearAttentionConfig, SlotStateCache, sequence_starts
from ..layers.rotary import DefaultRotaryEmbeddingsConfig, RotaryEmbeddingsConfig, rope_from_entry, rope_to_entry
from ..nn import Embedding, Linear
from ..ops.depth_stream import norm_of_depths, shift_tokens
from ..ops.glu import ClampedGlu
from ..ops.residual_stream import embed_stream, project
from ..utils.remat import ScanCheckpointPolicy, should_recompute
from .llama import LlamaMlp, RecurrentLMHeadModel
from .lm_model import LmConfig

MIXERS = ("lightning", "retention", "latent_attention")


@dataclass(frozen=True)
class MumizenLayerConfig:
    """Sizes of one layer.  Which fields count depends on ``mixer``:

    * lightning, retention: ``num_heads``, ``head_dim``, ``v_head_dim``, ``decay`` (one per head);
    * latent_attention: ``num_heads``, ``head_dim`` (the part without positions), ``rotary_dim`` (the rotated part, turned by ``rope``),
      ``v_head_dim``, ``q_lora_rank``, ``kv_lora_rank``, ``attention_scale``, ``kv_from`` (the layer whose latents it reads; None: its own).

    ``intermediate_dim`` is the feed-forward's (an expert's, when ``num_experts > 0``), with inputs bounded by ``limit``; None: the layer has
    no feed-forward.  ``shared_intermediate_dim`` None: no shared expert."""

    mixer: str = "lightning"
    num_heads: int = 16
    head_dim: int = 128
    v_head_dim: int = 128
    decay: Tuple[float, ...] = ()
    rotary_dim: int = 64
    rope: RotaryEmbeddingsConfig = field(default_factory=DefaultRotaryEmbeddingsConfig)
    q_lora_rank: int = 1536
    kv_lora_rank: int = 512
    attention_scale: float = 192 ** -0.5
    kv_from: Optional[int] = None
    intermediate_dim: Optional[int] = 8192
    limit: float = 7.0
    num_experts: int = 0
    num_experts_per_tok: int = 0
    shared_intermediate_dim: Optional[int] = None
    shared_limit: float = 7.0

    def __post_init__(self):
        if self.mixer not in MIXERS:
            raise ValueError(f"unknown mixer {self.mixer!r}: one of {', '.join(MIXERS)}")
        object.__setattr__(self, "decay", tuple(float(d) for d in self.decay))
        if self.mixer == "latent_attention":
            if self.kv_from is not None and self.kv_from < 0:
                raise ValueError("kv_from is the number of an earlier layer")
            if self.rope.build(self.rotary_dim).rotary_dim != self.rotary_dim:
                raise ValueError(f"the rotated part has {self.rotary_dim} dimensions and all of them turn")
        elif len(self.decay) != self.num_heads:
            raise ValueError(f"{len(self.decay)} decays for {self.num_heads} heads")
        if self.intermediate_dim is not None and self.num_experts > 0 and not 0 < self.num_experts_per_tok <= self.num_experts:
            raise ValueError(f"a token cannot use {self.num_experts_per_tok} of {self.num_experts} experts")

    @property
    def keeps(self) -> Tuple:
        """What has to agree between a layer and one that reads its latents."""
        return self.kv_lora_rank, self.rotary_dim, self.rope


def _layer_from_checkpoint(entry: dict) -> MumizenLayerConfig:
    kind, m, f = entry["type"], entry["mixer"], entry.get("mlp")
    kw = dict(mixer=kind, num_heads=m["heads"], head_dim=m["dim"], v_head_dim=m["vdim"], intermediate_dim=None)
    if kind == "latent_attention":
        if m["rot"]["dims"] != m["rot_dim"]:
            raise ValueError(f"the rotated part has {m['rot_dim']} dimensions but {m['rot']['dims']} of them are to rotate")
        kw.update(rotary_dim=m["rot_dim"], rope=rope_from_entry(m["rot"]), q_lora_rank=m["q_rank"], kv_lora_rank=m["kv_rank"],
                  attention_scale=float(m["scale"]), kv_from=m.get("kv_from"))
    elif kind in MIXERS:
        kw.update(decay=tuple(m["decay"]))
    if f is not None:
        if f["kind"] == "dense":
            kw.update(intermediate_dim=f["ff"], limit=float(f["limit"]))
        elif f["kind"] == "moe":
            shared = f.get("shared")
            kw.update(intermediate_dim=f["expert"]["ff"], limit=float(f["expert"]["limit"]), num_experts=f["router"]["experts"],
                      num_experts_per_tok=f["router"]["top"])
            if shared is not None:
                kw.update(shared_intermediate_dim=shared["ff"], shared_limit=float(shared["limit"]))
        else:
            raise ValueError(f"unknown feed-forward kind {f['kind']!r}")
    return MumizenLayerConfig(**kw)


def _layer_to_checkpoint(c: MumizenLayerConfig) -> dict:
    m = dict(heads=c.num_heads, dim=c.head_dim, vdim=c.v_head_dim)
    if c.mixer == "latent_attention":
        m.update(rot_dim=c.rotary_dim, rot=rope_to_entry(c.rope, c.rotary_dim), q_rank=c.q_lora_rank, kv_rank=c.kv_lora_rank, scale=c.attention_scale)
        if c.kv_from is not None:
            m["kv_from"] = c.kv_from
    else:
        m["decay"] = list(c.decay)
    mlp = None
    if c.intermediate_dim is not None:
        one = dict(ff=c.intermediate_dim, limit=c.limit)
        mlp = dict(kind="dense", **one) if c.num_experts == 0 else \
            dict(kind="moe", expert=one, router=dict(experts=c.num_experts, top=c.num_experts_per_tok))
        if c.num_experts > 0 and c.shared_intermediate_dim is not None:
            mlp["shared"] = dict(ff=c.shared_intermediate_dim, limit=c.shared_limit)
    return dict(type=c.mixer, mixer=m, mlp=mlp)


@LmConfig.register_subclass("mumizen")
@dataclass(frozen=True)
class MumizenConfig(HFCompatConfig):
    seq_len: int = 8192
    hidden_dim: int = 2048
    layer_norm_epsilon: float = 1e-5
    norm_groups: int = 1
    layers: Tuple[MumizenLayerConfig, ...] = (MumizenLayerConfig(decay=(0.99,) * 16),)
    initializer_range: float = 0.02
    upcast_attn: bool = False
    attn_backend: Optional[AttentionBackend] = None
    gradient_checkpointing: Union[bool, ScanCheckpointPolicy, str] = True
    reference_checkpoint: Optional[str] = None
    tokenizer: Optional[str] = None
    cross_entropy_block_size: Optional[int] = None

    hf_architecture = "Mumizen"
    hf_vocab_key = "vocab"
    tie_word_embeddings = False

    def __post_init__(self):
        layers = tuple(MumizenLayerConfig(**l) if isinstance(l, dict) else l for l in self.layers)
        object.__setattr__(self, "layers", layers)
        if not layers:
            raise ValueError("a model has at least one layer")
        if self.norm_groups <= 0 or self.hidden_dim % self.norm_groups != 0:
            raise ValueError(f"{self.hidden_dim} dimensions have no {self.norm_groups} equal groups")
        for i, l in enumerate(layers):
            if l.mixer != "latent_attention" or l.kv_from is None:
                continue
            j = layers[l.kv_from] if l.kv_from < i else None
            if j is None or j.mixer != "latent_attention" or j.kv_from is not None or j.keeps != l.keeps:
                raise ValueError(f"layer {i} cannot read the latents of layer {l.kv_from}")

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def model_type(self) -> Type["MumizenLMHeadModel"]:
        return MumizenLMHeadModel

    def hf_checkpoint_converter(self, ref_checkpoint: Optional[str] = None) -> HFCheckpointConverter:
        return HFCheckpointConverter(self.__class__, reference_checkpoint=ref_checkpoint or self.reference_checkpoint,
                                     tokenizer=ref_checkpoint if self.tokenizer is None else self.tokenizer)

    @classmethod
    def from_hf_config(cls, hf_config) -> "MumizenConfig":
        c = hf_config if isinstance(hf_config, dict) else vars(hf_config)
        return cls(hidden_dim=c["width"], layer_norm_epsilon=float(c["norm"]["eps"]), norm_groups=c["norm"]["groups"],
                   layers=tuple(_layer_from_checkpoint(l) for l in c["layers"]))

    def to_hf_config(self, vocab_size: int, config_overrides: Optional[Dict] = None) -> dict:
        cfg = dict(architecture=self.hf_architecture, vocab=vocab_size, width=self.hidden_dim,
                   norm={"eps": self.layer_norm_epsilon, "groups": self.norm_groups}, layers=[_layer_to_checkpoint(l) for l in self.layers])
        cfg.update(config_overrides or {})
        return cfg

    @property
    def norm_config(self) -> LayerNormConfigBase:
        return GroupedRmsNormConfig(eps=self.layer_norm_epsilon, groups=self.norm_groups)

    def mk_LayerNorm(self, dim: int):
        return self.norm_config.build(dim)

    def build_mixer(self, l: MumizenLayerConfig) -> nn.Module:
        std, eps = self.initializer_range, self.layer_norm_epsilon
        if l.mixer == "latent_attention":
            return MultiHeadLatentAttention(MultiHeadLatentAttentionConfig(
                hidden_dim=self.hidden_dim, num_heads=l.num_heads, kv_lora_rank=l.kv_lora_rank, q_lora_rank=l.q_lora_rank, qk_rope_head_dim=l.rotary_dim,
                qk_nope_head_dim=l.head_dim, v_head_dim=l.v_head_dim, upcast_attn=self.upcast_attn, attn_backend=self.attn_backend, rope=l.rope,
                scaling_factor=l.attention_scale, norm_eps=eps, output_gate=True, shares_latent=l.kv_from is not None), init_std=std)
        lightning = l.mixer == "lightning"
        return LinearAttention(LinearAttentionConfig(
            hidden_dim=self.hidden_dim, num_heads=l.num_heads, head_dim=l.head_dim, v_head_dim=l.v_head_dim, decay=l.decay,
            key_scale=1.0 if lightning else l.head_dim ** -0.5, silu=lightning, norm_per_head=not lightning, sigmoid_gate=lightning, norm_eps=eps), init_std=std)

    def build_feed_forward(self, l: MumizenLayerConfig) -> nn.Module:
        std = self.initializer_range
        if l.num_experts == 0:
            return LlamaMlp(self.hidden_dim, l.intermediate_dim, ClampedGlu(l.limit), init_std=std)
        return GroupedSoftmaxMoe(self.hidden_dim, l.intermediate_dim, l.num_experts, l.num_experts_per_tok, shared_intermediate=l.shared_intermediate_dim,
                                 shared_gated=False, activation=ClampedGlu(l.limit), shared_activation=ClampedGlu(l.shared_limit), router_bias=True,
                                 init_std=std)

    def _products(self, l: MumizenLayerConfig, active: bool) -> int:
        """Weights of a layer's matrix products (``active``: of those that a token uses)."""
        e, H, d, dv = self.hidden_dim, l.num_heads, l.head_dim, l.v_head_dim
        n = 2 * e * H * dv  # gate and output
        if l.mixer == "latent_attention":
            n += l.q_lora_rank * (e + H * (d + l.rotary_dim)) + l.kv_lora_rank * H * (d + dv)
            n += 0 if l.kv_from is not None else e * (l.kv_lora_rank + l.rotary_dim)
        else:
            n += e * H * (2 * d + dv)
        if l.intermediate_dim is not None:
            if l.num_experts == 0:
                return n + 3 * e * l.intermediate_dim
            n += e * l.num_experts + 3 * e * l.intermediate_dim * (l.num_experts_per_tok if active else l.num_experts)
            n += 3 * e * (l.shared_intermediate_dim or 0)
        return n

    def flops_per_token(self, vocab_size: int) -> float:
        flops = 2.0 * vocab_size * self.hidden_dim
        for l in self.layers:
            flops += 2.0 * self._products(l, True)
            flops += 2 * l.num_heads * (l.head_dim + l.rotary_dim + l.v_head_dim) * self.seq_len if l.mixer == "latent_attention" \
                else 4 * l.num_heads * l.head_dim * l.v_head_dim
        return flops

    def total_trainable_params(self, vocab_size: int) -> int:
        e = self.hidden_dim
        n = e + 2 * vocab_size * e
        for i, l in enumerate(self.layers):
            n += self._products(l, False) + (2 * e if l.intermediate_dim is None else 3 * e) + i + 2  # norms, shift; depth weights
            if l.mixer == "latent_attention":
                n += l.q_lora_rank + (0 if l.kv_from is not None else l.kv_lora_rank)
            elif l.mixer == "lightning":
                n += l.num_heads * l.v_head_dim
            n += 0 if l.intermediate_dim is None else l.num_experts  # router bias
        return n


@dataclass
class MumizenLayerCache:
    """What a layer keeps: ``mixer`` (pages, or state by slot; None: it reads an earlier layer's pages) and ``shift``, the last normed row of
    every slot."""

    mixer: object
    shift: SlotStateCache

    def copy_page(self, src_page: int, dst_page: int) -> "MumizenLayerCache":
        if self.mixer is not None:
            self.mixer.copy_page(src_page, dst_page)
        return self

    def copy_slot(self, src: int, dst: int) -> "MumizenLayerCache":
        if self.mixer is not None:
            self.mixer.copy_slot(src, dst)
        self.shift.copy_slot(src, dst)
        return self


class MumizenDecoderLayer(nn.Module):
    """``x`` is the fp32 stream that the layer starts from; ``shift`` mixes a token's normed row with the one before it, and ``depth_weights``
    average the results of the layers up to this one."""

    def __init__(self, config: MumizenConfig, layer: MumizenLayerConfig, index: int):
        super().__init__()
        e = config.hidden_dim
        self.kind, self.kv_from = layer.mixer, layer.kv_from
        self.mixer = config.build_mixer(layer)
        self.input_layernorm = config.mk_LayerNorm(e)
        self.shift = nn.Parameter(torch.full((e,), 0.25))
        self.shift.lev_shape = (e,)
        self.depth_weights = nn.Parameter(torch.zeros(index + 2))
        self.depth_weights.lev_shape = (index + 2,)
        if self.depth_weights.device.type != "meta":
            with torch.no_grad():
                self.depth_weights[-1] = 1.0
        self.mlp = None
        if layer.intermediate_dim is not None:
            self.post_mixer_layernorm = config.mk_LayerNorm(e)
            self.mlp = config.build_feed_forward(layer)

    def _feed_forward(self, x, batch_info=None):
        if self.mlp is None:
            return x
        return self.mlp.add_to_stream(x, self.post_mixer_layernorm.from_stream(x), batch_info)

    def forward(self, x, mask=None, pos_ids=None, kept=None):
        """``(result, kept)``: ``kept`` is what a later layer may read of this one's latents, or what this one reads of an earlier one's."""
        h = shift_tokens(self.input_layernorm.in_fp32(x), self.shift, sequence_starts(mask)).to(self.input_layernorm.weight.dtype)
        if self.kind == "latent_attention":
            y, kept = self.mixer.forward_sharing(h, mask, pos_ids, kept)
        else:
            y = self.mixer(h, mask, pos_ids)
        return self._feed_forward(x + y.float()), kept


class MumizenTransformer(nn.Module):
    def __init__(self, config: MumizenConfig):
        super().__init__()
        self.config = config
        self.layers = nn.ModuleList([MumizenDecoderLayer(config, l, i) for i, l in enumerate(config.layers)])
        self.norm = config.mk_LayerNorm(config.hidden_dim)

    def forward(self, x, mask=None, pos_ids=None):
        remat = should_recompute(self.config.gradient_checkpointing) and torch.is_grad_enabled() and self.training
        history, kept = [x], {}
        for i, layer in enumerate(self.layers):
            args = (x, mask, pos_ids, kept.get(layer.kv_from))
            y, kept[i] = checkpoint(layer, *args, use_reentrant=False) if remat else layer(*args)
            history.append(y)
            x = sum(w * t for w, t in zip(layer.depth_weights.float(), history))
        return self.norm.from_stream(x)

    @torch.no_grad()
    def decode(self, history, caches, batch_info, pos_ids, logit_rows=None):
        """``history [layers + 1, T, hidden]`` fp32: the first plane holds the embeddings, layer ``i`` leaves its result in plane ``i + 1``."""
        eps, groups = self.config.layer_norm_epsilon, self.config.norm_groups
        coef, latents = None, {}
        for i, (layer, cache) in enumerate(zip(self.layers, caches)):
            stream = history[i + 1]
            h = norm_of_depths(history[:i + 1], layer.input_layernorm.weight, eps, groups=groups, coef=coef, out=stream, shift=layer.shift,
                               state=cache.shift.state, batch_info=batch_info)
            if layer.kind == "latent_attention":
                j = i if layer.kv_from is None else layer.kv_from
                x, latents[i] = layer.mixer.paged_decode_stream_sharing(h, caches[j].mixer, batch_info, pos_ids, stream, latents.get(j))
            else:
                x, _ = layer.mixer.paged_decode_stream(h, cache.mixer, batch_info, pos_ids, stream)
            x = layer._feed_forward(x, batch_info)
            if x.data_ptr() != stream.data_ptr():  # steps that could not accumulate in place
                stream.copy_(x)
            coef = layer.depth_weights
        return norm_of_depths(history, self.norm.weight, eps, groups=groups, coef=coef, rows=logit_rows), caches

    def initial_cache(self, max_pages: int, page_size: int, max_seqs: int, *, dtype=torch.bfloat16, device=None):
        def mixer_cache(l):
            if l.kind != "latent_attention":
                return l.mixer.empty_state(max_seqs, device=device)
            return None if l.kv_from is not None else l.mixer.empty_page_cache(max_pages, page_size, dtype=dtype, device=device)

        return [MumizenLayerCache(mixer_cache(l), SlotStateCache.init(max_seqs, self.config.hidden_dim, device=device)) for l in self.layers]


class MumizenEmbedding(nn.Module):
    def __init__(self, vocab_size: int, config: MumizenConfig):
        super().__init__()
        self.token_embeddings = Embedding(vocab_size, config.hidden_dim, init_std=config.initializer_range)

    def embed(self, input_ids, out=None):
        return embed_stream(input_ids, self.token_embeddings.weight, 1.0, out=out)

    forward = embed


class MumizenLMHeadModel(RecurrentLMHeadModel):
    """Shares the vocabulary handling of the Llama head model."""

    def __init__(self, vocab_size: int, config: MumizenConfig, *, tp=None):
        nn.Module.__init__(self)
        if tp is not None and tp.size > 1:
            raise NotImplementedError("mumizen has no tensor-parallel form")
        self.config = config
        self._vocab_size = vocab_size
        self.transformer = MumizenTransformer(config)
        self.embeddings = MumizenEmbedding(vocab_size, config)
        self.lm_head = Linear(config.hidden_dim, vocab_size, init_std=config.initializer_range)

    def activations(self, input_ids, attn_mask=None, *, pos_ids=None):
        return self.transformer(self.embeddings.embed(input_ids), attn_mask if attn_mask is not None else AttentionMask.causal(), pos_ids)

    def decode(self, input_ids, kv_cache, batch_info, pos_ids, logit_rows: Optional[torch.Tensor] = None):
        w = self.embeddings.token_embeddings.weight
        history = torch.empty(self.config.num_layers + 1, input_ids.numel(), self.config.hidden_dim, dtype=torch.float32, device=w.device)
        self.embeddings.embed(input_ids, out=history[0])
        h, kv_cache = self.transformer.decode(history, kv_cache, batch_info, pos_ids, logit_rows)
        return project(h, self.get_lm_head(), out_dtype=torch.float32), kv_cache

    # -- checkpoint names ----------------------------------------------------------------------------------------
    def hf_tensor_parts(self, name: str, t: torch.Tensor) -> List[Tuple[str, torch.Tensor, Tuple[int, ...]]]:
        """``(checkpoint tensor, view of t, its shape in the checkpoint)`` of a parameter's value ``t``."""
        top = {"embeddings.token_embeddings.weight": "embed", "lm_head.weight": "head", "transformer.norm.weight": "final.norm"}
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
        fixed = {"input_layernorm.weight": "norm1", "post_mixer_layernorm.weight": "norm2", "shift": "shift", "depth_weights": "dwa",
                 "mixer.q_a_proj.weight": "mix.dq", "mixer.q_a_norm.weight": "mix.dq.norm", "mixer.q_b_proj.weight": "mix.uq",
                 "mixer.kv_a_proj.weight": "mix.dkv", "mixer.kv_a_norm.weight": "mix.dkv.norm", "mixer.o_norm.weight": "mix.norm",
                 "mlp.router.weight": "mlp.router", "mlp.router.bias": "mlp.router.b"}
        if rest in fixed:
            return [(pre + fixed[rest], t, t.shape)]
        owner, proj, _ = rest.rsplit(".", 2)  # mixer.{q,k,v,g,o}_proj, mlp.{gate,up,down}_proj, mlp.shared.{gate,up,down}_proj
        return [(f"{pre}{owner.replace('mixer', 'mix')}.{proj[:-len('_proj')]}", t, t.shape)]
