"""Attention: structured masks, the dispatching ``dot_product_attention``, the ``Attention`` module with
GQA / qk-norm / RoPE / sinks, multi-head latent attention, and the paged KV cache used by the inference engine.

Reference behaviour: src/levanter/layers/attention.py (mask :757-1003, dispatch :71-241, vanilla :329-378,
sink :244-326, module :1373-1635, KvPageCache :1638-1707, ragged paged attention :1710-1991, MLA :1994-2213).

Tensor layout here is ``q[B, Sq, Hq, D]``, ``k/v[B, Sk, Hkv, D]`` with ``Hq = Hkv * q_per_kv`` and query head
``h`` reading KV head ``h // q_per_kv`` (the reference's ``(kv_head, q_heads_per_group)`` articulation).
"""
from __future__ import annotations

import enum
import math
from dataclasses import dataclass, field, replace
from typing import Optional, Tuple, Union

import torch
import torch.nn as nn
import torch.nn.functional as F

from .normalization import LayerNormConfigBase, RmsNormConfig
from .rotary import DefaultRotaryEmbeddingsConfig, RotaryEmbeddings, RotaryEmbeddingsConfig


class AttentionBackend(str, enum.Enum):
    DEFAULT = "default"      # B200 flash kernel on a B200, blockwise PyTorch elsewhere
    B200 = "b200"            # hand-written sm_100a flash attention (ops.flash_attention)
    TORCH_FLASH = "torch_flash"  # blockwise FA-2 in PyTorch ops (counterpart of the reference's JAX_FLASH)
    SDPA = "sdpa"            # torch.nn.functional.scaled_dot_product_attention (library kernel; baseline/oracle)
    VANILLA = "vanilla"      # materialise the score matrix
    # names accepted from reference configs; they select DEFAULT here
    NVTE = "nvte"
    SPLASH = "splash"
    JAX_FLASH = "jax_flash"


# --------------------------------------------------------------------------------------------- masks
def _and(a, b):
    if a is None:
        return b
    if b is None:
        return a
    return a & b


def _or(a, b):
    if a is None or b is None:
        return None if (a is None and b is None) else (a if b is None else b)
    return a | b


def causal_mask(q_len: int, k_len: int, q_start=0, k_start=0, device=None) -> torch.Tensor:
    qp = torch.arange(q_len, device=device) + q_start
    kp = torch.arange(k_len, device=device) + k_start
    return qp[:, None] >= kp[None, :]


def chunk_segments(segment_ids: torch.Tensor, chunk_size: int) -> torch.Tensor:
    """Segment ids ``[..., S]`` cut further into chunks of ``chunk_size`` positions, counted from the start of each run of equal
    ids: non-decreasing ids, one per (run, chunk).  Negative ids (padding) stay as they are."""
    S = segment_ids.shape[-1]
    idx = torch.arange(S, device=segment_ids.device).expand(segment_ids.shape)
    new_run = torch.ones_like(segment_ids, dtype=torch.bool)
    new_run[..., 1:] = segment_ids[..., 1:] != segment_ids[..., :-1]
    start = torch.where(new_run, idx, torch.zeros_like(idx)).cummax(dim=-1).values
    out = torch.cumsum((idx - start) % chunk_size == 0, dim=-1) - 1
    return torch.where(segment_ids < 0, segment_ids.to(out.dtype), out)


@dataclass(frozen=True)
class AttentionMask:
    """Conjunction of structured masks: causal (with an optional offset), explicit, sliding window, segment ids, chunks.

    ``materialize(q_len, k_len, q_slice, k_slice)`` returns the boolean mask of a block so block-wise kernels
    can skip or specialise blocks (src/levanter/layers/attention.py:795-846)."""

    is_causal: bool = False
    causal_offset: Union[None, int, torch.Tensor] = None
    explicit_mask: Optional[torch.Tensor] = None            # [..., Sq, Sk] bool
    segment_ids: Optional[Tuple[torch.Tensor, torch.Tensor]] = None  # ([B, Sq], [B, Sk])
    sliding_window: Optional[int] = None
    segments_sorted: bool = False
    """the segment ids are non-decreasing along the sequence with negative ids (padding) only at the end, as in packed
    batches: kernels may then skip every key block that lies before a query block's first sequence"""
    chunk_size: Optional[int] = None
    """positions are cut into chunks of this size, counted from the start of the sequence (of the segment, with segment ids), and a
    query sees the keys of its own chunk only; queries and keys must be the same positions"""

    def __post_init__(self):
        if self.segment_ids is not None and not isinstance(self.segment_ids, tuple):
            object.__setattr__(self, "segment_ids", (self.segment_ids, self.segment_ids))

    @staticmethod
    def causal(*, sliding_window: Optional[int] = None, offset=None) -> "AttentionMask":
        return AttentionMask(is_causal=True, causal_offset=offset, sliding_window=sliding_window)

    @staticmethod
    def explicit(mask: torch.Tensor) -> "AttentionMask":
        return AttentionMask(is_causal=False, explicit_mask=mask)

    def with_segment_ids(self, segment_ids, kv_segment_ids=None, *, sorted: bool = False) -> "AttentionMask":
        return replace(self, segment_ids=(segment_ids, segment_ids if kv_segment_ids is None else kv_segment_ids),
                       segments_sorted=bool(sorted))

    def with_chunk_size(self, chunk_size: Optional[int]) -> "AttentionMask":
        return replace(self, chunk_size=chunk_size)

    def chunks_as_segments(self) -> "AttentionMask":
        """The same mask without a chunk size: chunks expressed as segment ids (needs segment ids to start from)."""
        if self.chunk_size is None:
            return self
        seg = chunk_segments(self.segment_ids[0], self.chunk_size)
        return replace(self, segment_ids=(seg, seg), chunk_size=None)

    def with_sliding_window(self, sliding_window: Optional[int]) -> "AttentionMask":
        return replace(self, sliding_window=sliding_window)

    def materialize(self, q_len: int, k_len: int, q_slice: Optional[Tuple[int, int]] = None,
                    k_slice: Optional[Tuple[int, int]] = None, device=None) -> Optional[torch.Tensor]:
        """Boolean mask broadcastable to ``[B, 1, q, k]`` for the block ``q_slice=(start,size)`` x ``k_slice``."""
        qs, qn = q_slice if q_slice is not None else (0, q_len)
        ks, kn = k_slice if k_slice is not None else (0, k_len)
        mask = None
        if self.is_causal:
            off = 0 if self.causal_offset is None else self.causal_offset
            if isinstance(off, torch.Tensor) and off.dim() > 0:
                qp = (torch.arange(qn, device=device) + qs)[None, :, None]
                kp = (torch.arange(kn, device=device) + ks)[None, None, :]
                mask = (qp + off.to(device).view(-1, 1, 1) >= kp).unsqueeze(1)
            else:
                off = int(off)
                mask = causal_mask(qn, kn, qs, ks - off, device)
        if self.explicit_mask is not None:
            em = self.explicit_mask[..., qs:qs + qn, ks:ks + kn]
            if em.dim() == 3:
                em = em.unsqueeze(1)
            mask = _and(mask, em.to(torch.bool))
        if self.sliding_window is not None:
            qp = torch.arange(qn, device=device) + qs
            kp = torch.arange(kn, device=device) + ks
            diff = qp[:, None] - kp[None, :]
            mask = _and(mask, (diff >= 0) & (diff < self.sliding_window))
        if self.segment_ids is not None:
            qseg, kseg = self.segment_ids if self.chunk_size is None else self.chunks_as_segments().segment_ids
            sm = qseg[..., qs:qs + qn, None] == kseg[..., None, ks:ks + kn]
            if sm.dim() == 3:
                sm = sm.unsqueeze(1)
            mask = _and(mask, sm)
        elif self.chunk_size is not None:
            qp = torch.arange(qn, device=device) + qs
            kp = torch.arange(kn, device=device) + ks
            mask = _and(mask, (qp // self.chunk_size)[:, None] == (kp // self.chunk_size)[None, :])
        return mask

    def __and__(self, other: "AttentionMask") -> "AttentionMask":
        if self.is_causal and other.is_causal:
            if self.causal_offset is not None and other.causal_offset is not None:
                same = self.causal_offset == other.causal_offset
                if isinstance(same, torch.Tensor):
                    same = bool(same.all())
                if not same:
                    raise ValueError("Mismatched causal offsets cannot be combined with &")
                offset = self.causal_offset
            else:
                offset = self.causal_offset if self.causal_offset is not None else other.causal_offset
            is_causal = True
        elif self.is_causal:
            is_causal, offset = True, self.causal_offset
        elif other.is_causal:
            is_causal, offset = True, other.causal_offset
        else:
            is_causal, offset = False, None
        if self.sliding_window is None:
            sw = other.sliding_window
        elif other.sliding_window is None:
            sw = self.sliding_window
        else:
            sw = min(self.sliding_window, other.sliding_window)
        if self.chunk_size is not None and other.chunk_size is not None and self.chunk_size != other.chunk_size:
            raise ValueError("Different chunk sizes cannot be combined with &")
        chunk = self.chunk_size if self.chunk_size is not None else other.chunk_size
        return AttentionMask(is_causal, offset, _and(self.explicit_mask, other.explicit_mask), self._same_segments(other), sw, chunk_size=chunk)

    def __or__(self, other: "AttentionMask") -> "AttentionMask":
        if self.chunk_size != other.chunk_size:
            raise ValueError("Different chunk sizes cannot be combined with |")

        def same_off():
            if self.causal_offset is None and other.causal_offset is None:
                return True
            if self.causal_offset is None or other.causal_offset is None:
                return False
            s = self.causal_offset == other.causal_offset
            return bool(s.all()) if isinstance(s, torch.Tensor) else bool(s)

        if self.is_causal and other.is_causal and same_off():
            is_causal, offset = True, self.causal_offset
        else:
            is_causal, offset = False, None
        if self.sliding_window is None or other.sliding_window is None:
            sw = None
        else:
            sw = max(self.sliding_window, other.sliding_window)
        return AttentionMask(is_causal, offset, _or(self.explicit_mask, other.explicit_mask), self._same_segments(other), sw,
                             chunk_size=self.chunk_size)

    def _same_segments(self, other):
        a, b = self.segment_ids, other.segment_ids
        if a is not None and b is not None:
            if not (torch.equal(a[0], b[0]) and torch.equal(a[1], b[1])):
                raise ValueError("Only one segment mask is allowed")
            return a
        return a if a is not None else b


def materialize_mask(mask: Union[None, torch.Tensor, AttentionMask], q_len: int, k_len: int, device=None,
                     q_slice=None, k_slice=None) -> Optional[torch.Tensor]:
    if mask is None:
        return None
    if isinstance(mask, AttentionMask):
        return mask.materialize(q_len, k_len, q_slice, k_slice, device=device)
    qs, qn = q_slice if q_slice is not None else (0, q_len)
    ks, kn = k_slice if k_slice is not None else (0, k_len)
    m = mask[..., qs:qs + qn, ks:ks + kn]
    if m.dim() == 3:
        m = m.unsqueeze(1)
    return m


# --------------------------------------------------------------------------------------------- attention functions
def _expand_kv(k: torch.Tensor, q_heads: int) -> torch.Tensor:
    kv = k.shape[2]
    if kv == q_heads:
        return k
    return k.repeat_interleave(q_heads // kv, dim=2)


def simple_attention_with_dropout(q, k, v, mask=None, bias=None, *, dropout: float = 0.0, inference: bool = True,
                                  attention_dtype: Optional[torch.dtype] = None, logits_soft_cap: Optional[float] = None,
                                  scaling_factor: Optional[float] = None) -> torch.Tensor:
    """Vanilla attention: scale q, QK^T, +bias, tanh soft-cap, mask -> -1e9, softmax in ``attention_dtype``, dropout, .V
    (src/levanter/layers/attention.py:329-378)."""
    B, Sq, H, D = q.shape
    Sk = k.shape[1]
    scale = scaling_factor if scaling_factor is not None else 1.0 / math.sqrt(D)
    orig = v.dtype
    kk = _expand_kv(k, H)
    vv = _expand_kv(v, H)
    if attention_dtype is not None:
        q, kk = q.to(attention_dtype), kk.to(attention_dtype)
    w = torch.einsum("bqhd,bkhd->bhqk", q * scale, kk)
    if bias is not None:
        w = w + bias
    if logits_soft_cap is not None:
        w = torch.tanh(w / logits_soft_cap) * logits_soft_cap
    m = materialize_mask(mask, Sq, Sk, device=q.device)
    if m is not None:
        w = torch.where(m, w, torch.full_like(w, -1e9))
    w = torch.softmax(w.float() if attention_dtype is None else w, dim=-1).to(orig)
    if dropout > 0.0 and not inference:
        w = F.dropout(w, dropout, training=True)
    return torch.einsum("bhqk,bkhd->bqhd", w, vv)


def _structured_only(mask) -> bool:
    """True when the mask has only the structures the fused kernels understand natively."""
    if mask is None:
        return True
    if not isinstance(mask, AttentionMask):
        return False
    if mask.explicit_mask is not None:
        return False
    if mask.causal_offset is not None and not (isinstance(mask.causal_offset, int) and mask.causal_offset == 0):
        off = mask.causal_offset
        if isinstance(off, torch.Tensor) and off.dim() == 0 and int(off) == 0:
            return True
        return False
    return True


def dot_product_attention(q, k, v, mask: Union[None, torch.Tensor, AttentionMask] = None, bias=None, *,
                          attention_dtype: Optional[torch.dtype] = None, dropout: float = 0.0, inference: bool = True,
                          use_flash: Optional[bool] = None, attn_backend: Optional[AttentionBackend] = None,
                          flash_block_size: Optional[int] = None, logits_soft_cap: Optional[float] = None,
                          scaling_factor: Optional[float] = None) -> torch.Tensor:
    """Dispatch to the best available attention implementation (src/levanter/layers/attention.py:71-241).

    On a B200 the default is the hand-written flash kernel whenever the mask is structured (causal / sliding
    window / segment ids), there is no bias and no dropout; anything else falls through to blockwise PyTorch
    flash attention and finally to the vanilla implementation."""
    from ..models import flash_attention as FA
    from ..ops import flash_attention as KFA

    backend = attn_backend or AttentionBackend.DEFAULT
    if isinstance(backend, str) and not isinstance(backend, AttentionBackend):
        backend = AttentionBackend(backend)
    if backend in (AttentionBackend.NVTE, AttentionBackend.SPLASH):
        backend = AttentionBackend.DEFAULT
    if backend == AttentionBackend.JAX_FLASH:
        backend = AttentionBackend.TORCH_FLASH
    if use_flash is False:
        backend = AttentionBackend.VANILLA
    no_drop = dropout == 0.0 or inference

    if backend in (AttentionBackend.DEFAULT, AttentionBackend.B200):
        if KFA.supported(q, k, v, mask, bias, no_drop, attention_dtype):
            return KFA.flash_attention(q, k, v, mask, logits_soft_cap=logits_soft_cap, scaling_factor=scaling_factor)
        if backend == AttentionBackend.B200:
            raise ValueError("the B200 flash-attention kernel does not support this call (bias, dropout, explicit mask, dtype or head size)")
        plain = mask is None or (isinstance(mask, AttentionMask) and mask.explicit_mask is None and mask.segment_ids is None
                                 and mask.sliding_window is None and mask.chunk_size is None and _structured_only(mask)) \
            and v.shape[-1] == q.shape[-1]
        if q.is_cuda and plain and bias is None and no_drop and logits_soft_cap is None and q.dtype in (torch.bfloat16, torch.float16) \
                and q.shape[1] == k.shape[1]:
            # shapes the tcgen05 kernels do not cover (head sizes other than 64 and 128, cross attention): the library's fused
            # attention rather than the blockwise PyTorch loop
            backend = AttentionBackend.SDPA
        else:
            backend = AttentionBackend.TORCH_FLASH if q.shape[1] > 1 else AttentionBackend.VANILLA

    if backend == AttentionBackend.SDPA and bias is None and no_drop and logits_soft_cap is None:
        B, Sq, H, D = q.shape
        m = materialize_mask(mask, Sq, k.shape[1], device=q.device)
        is_causal = isinstance(mask, AttentionMask) and mask.is_causal and mask.explicit_mask is None and \
            mask.segment_ids is None and mask.sliding_window is None and mask.chunk_size is None and _structured_only(mask)
        out = F.scaled_dot_product_attention(
            q.transpose(1, 2), _expand_kv(k, H).transpose(1, 2), _expand_kv(v, H).transpose(1, 2),
            attn_mask=None if is_causal else m, is_causal=is_causal, scale=scaling_factor)
        return out.transpose(1, 2)

    if backend == AttentionBackend.TORCH_FLASH and bias is None and v.shape[-1] == q.shape[-1]:
        block = flash_block_size or FA.BLOCK_SIZE
        if q.shape[1] >= block and k.shape[1] >= block and q.shape[1] % block == 0 and k.shape[1] % block == 0:
            return FA.flash_attention(q, k, v, mask, dropout=dropout, inference=inference, block_size=block,
                                      dtype=attention_dtype, logits_soft_cap=logits_soft_cap, scaling_factor=scaling_factor)
    return simple_attention_with_dropout(q, k, v, mask, bias, dropout=dropout, inference=inference,
                                         attention_dtype=attention_dtype, logits_soft_cap=logits_soft_cap,
                                         scaling_factor=scaling_factor)


def dot_product_attention_with_sink(q, k, v, sink: torch.Tensor, mask=None, bias=None, **kw) -> torch.Tensor:
    """Attention with a learned per-head sink logit: a zero K/V column is appended and the sink logit is placed in
    the bias at that column (src/levanter/layers/attention.py:244-326).  ``sink``: ``[Hq]``."""
    B, Sq, H, D = q.shape
    Sk = k.shape[1]
    from ..ops import flash_attention as KFA

    if (kw.get("dropout", 0.0) == 0.0 or kw.get("inference", False)) and KFA.supported(q, k, v, mask, bias, True, kw.get("attention_dtype")):
        # the fused kernel takes the sink as one more term of the softmax denominator
        return KFA.flash_attention(q, k, v, mask, logits_soft_cap=kw.get("logits_soft_cap"), scaling_factor=kw.get("scaling_factor"),
                                   sink=sink)
    zk = torch.zeros(B, 1, k.shape[2], D, dtype=k.dtype, device=k.device)
    k2 = torch.cat([k, zk], dim=1)
    v2 = torch.cat([v, torch.zeros_like(zk)], dim=1)
    b = torch.zeros(B, H, Sq, Sk + 1, dtype=torch.float32, device=q.device)
    if bias is not None:
        b[..., :Sk] = bias
    b[..., Sk] = sink.float().view(1, H, 1)
    m = materialize_mask(mask, Sq, Sk, device=q.device)
    if m is not None:
        m = m.expand(B, -1, Sq, Sk) if m.dim() == 4 else m.expand(Sq, Sk)[None, None].expand(B, 1, Sq, Sk)
        m = torch.cat([m, torch.ones(B, m.shape[1], Sq, 1, dtype=torch.bool, device=q.device)], dim=-1)
    kw.pop("attn_backend", None)
    return simple_attention_with_dropout(q, k2, v2, m, b, **{k_: v_ for k_, v_ in kw.items() if k_ in
                                          ("dropout", "inference", "attention_dtype", "logits_soft_cap", "scaling_factor")})


# --------------------------------------------------------------------------------------------- module
from ..nn import FusedRows, Linear, RmsNorm  # noqa: E402  (after function definitions to keep the file readable)


@dataclass(frozen=True)
class AttentionConfig:
    """Configuration of the shared attention module (src/levanter/layers/attention.py:1373-1447)."""

    hidden_dim: int
    num_heads: int
    num_kv_heads: int
    head_dim: Optional[int] = None
    use_bias: bool = False
    use_output_bias: Optional[bool] = None
    upcast_attn: bool = False
    attn_backend: Optional[AttentionBackend] = None
    flash_attention_block_size: Optional[int] = None
    rope: Optional[RotaryEmbeddingsConfig] = None
    scaling_factor: Optional[float] = None
    logits_soft_cap: Optional[float] = None
    qk_norm: Optional[LayerNormConfigBase] = None
    sliding_window: Optional[int] = None
    v_head_dim: Optional[int] = None          # value size per head where it differs from the query/key size
    attention_chunk_size: Optional[int] = None  # a query sees its own chunk of that many positions only
    output_gate: bool = False                 # the heads are multiplied by sigmoid(W_g x) before the output projection
    head_temperature: bool = False            # a learned number per query head multiplies its scores
    value_mixing: bool = False                # v <- (1 - m) v + m v_first with a learned m and the first such layer's values
    head_gate: bool = False                   # head h is multiplied by sigmoid((W_g x)_h), one number per head (no bias)
    differential: Optional[float] = None      # two score maps per head over the same values, combined as in MapDifference; the number is the
    #                                           constant part of the second map's weight
    norm_eps: float = 1e-6                    # of the norm after the difference

    def __post_init__(self):
        assert self.num_heads % self.num_kv_heads == 0, "num_heads must be divisible by num_kv_heads"
        if self.differential is not None and (self.qk_norm is not None or self.head_temperature or self.output_gate):
            raise ValueError("differential attention takes neither qk_norm, nor head temperatures, nor a gate per element")
        if self.head_gate and self.output_gate:
            raise ValueError("a gate per head and a gate per element exclude each other")

    @property
    def maps(self) -> int:
        """Score maps per head."""
        return 1 if self.differential is None else 2

    @property
    def head_size(self) -> int:
        return self.head_dim if self.head_dim is not None else self.hidden_dim // self.num_heads

    @property
    def v_head_size(self) -> int:
        return self.v_head_dim if self.v_head_dim is not None else self.head_size

    @property
    def q_heads_per_group(self) -> int:
        return self.num_heads // self.num_kv_heads

    @property
    def use_flash_attention(self) -> bool:
        return self.attn_backend != AttentionBackend.VANILLA


class Attention(nn.Module):
    """Multi-head / grouped-query attention with optional per-head qk-norm and RoPE.

    Parameter layouts for checkpoints: ``q_proj.weight [kv_head, q_heads_per_group, head_size, embed]``,
    ``k_proj/v_proj.weight [kv_head, head_size, embed]``, ``o_proj.weight [embed, heads, head_size]``
    (src/levanter/layers/attention.py:1473-1488).  In memory they are the 2-D ``[out, in]`` matrices the GEMM
    kernels consume; the articulated shape is a reshape."""

    def __init__(self, config: AttentionConfig, *, init_std: float = 0.02, tp=None):
        super().__init__()
        c = config
        self.config = c
        D, Dv = c.maps * c.head_size, c.v_head_size
        self.tp = tp
        tp_size = tp.size if tp is not None else 1
        assert c.num_kv_heads % tp_size == 0 or tp_size == 1, "kv heads must divide the tensor-parallel size"
        self.local_heads = c.num_heads // tp_size
        self.local_kv = c.num_kv_heads // tp_size
        out_bias = c.use_output_bias if c.use_output_bias is not None else c.use_bias
        self.q_proj = Linear(c.hidden_dim, self.local_heads * D, bias=c.use_bias, init_std=init_std,
                             lev_out=(self.local_kv, c.q_heads_per_group, D), lev_in=(c.hidden_dim,), parallel=("column", tp))
        self.k_proj = Linear(c.hidden_dim, self.local_kv * D, bias=c.use_bias, init_std=init_std,
                             lev_out=(self.local_kv, D), lev_in=(c.hidden_dim,), parallel=("column", tp))
        self.v_proj = Linear(c.hidden_dim, self.local_kv * Dv, bias=c.use_bias, init_std=init_std,
                             lev_out=(self.local_kv, Dv), lev_in=(c.hidden_dim,), parallel=("column", tp))
        self.o_proj = Linear(self.local_heads * Dv, c.hidden_dim, bias=out_bias, init_std=init_std,
                             lev_out=(c.hidden_dim,), lev_in=(self.local_heads, Dv), parallel=("row", tp))
        if c.output_gate:
            self.g_proj = Linear(c.hidden_dim, self.local_heads * Dv, bias=c.use_bias, init_std=init_std,
                                 lev_out=(self.local_kv, c.q_heads_per_group, Dv), lev_in=(c.hidden_dim,), parallel=("column", tp))
        if c.head_gate:
            self.g_proj = Linear(c.hidden_dim, self.local_heads, init_std=init_std, lev_out=(self.local_kv, c.q_heads_per_group), lev_in=(c.hidden_dim,),
                                 parallel=("column", tp))
        if c.differential is not None:
            for n in self.difference_names:
                p = nn.Parameter(torch.randn(c.head_size) * 0.1)
                p.lev_shape = (c.head_size,)
                setattr(self, n, p)
            self._difference = None
        if c.qk_norm is not None:
            self.q_norm = c.qk_norm.build(D)
            self.k_norm = c.qk_norm.build(D)
        else:
            self.q_norm = None
            self.k_norm = None
        self.rot: Optional[RotaryEmbeddings] = c.rope.build(c.head_size) if c.rope is not None else None
        if c.head_temperature:
            self.temperature = nn.Parameter(torch.ones(self.local_heads))
            self.temperature.lev_shape = (self.local_heads,)
        if c.value_mixing:
            self.value_mix = nn.Parameter(torch.tensor(0.5))
            self.value_mix.lev_shape = ()
        rows = sum(m.weight.shape[0] for m in self._projections())
        pad = -rows % 8  # whole groups of 8 columns keep the slices of the joint product aligned
        self._rows, self._bias_rows = FusedRows(pad), FusedRows(pad + (self.local_heads if c.head_gate else 0))

    difference_names = ("lambda_q1", "lambda_k1", "lambda_q2", "lambda_k2")

    def _projections(self):
        return [self.q_proj, self.k_proj, self.v_proj] + ([self.g_proj] if self.config.output_gate or self.config.head_gate else [])

    # -- projections shared by training and paged decode (src/levanter/layers/attention.py:1606-1635)
    def _compute_qkv(self, x: torch.Tensor, pos_ids: Optional[torch.Tensor], rotate: bool = True):
        c = self.config
        D = c.head_size
        lead = x.shape[:-1]
        q = self.q_proj(x).view(*lead, c.maps * self.local_heads, D)
        k = self.k_proj(x).view(*lead, c.maps * self.local_kv, D)
        v = self.v_proj(x).view(*lead, self.local_kv, c.v_head_size)
        if self.q_norm is not None:
            q = self.q_norm(q)
            k = self.k_norm(k)
        if self.rot is not None and rotate:
            from ..ops import rope as rope_op

            q, k = rope_op.apply_rope(q, k, self.rot, pos_ids)
        return q, k, v

    def map_difference(self):
        """How the two score maps of a head are combined when serving (``ops.map_difference``); the weight of the second map is derived from
        the learned vectors and made again when one of them has moved or changed, and after every change of mode."""
        from ..ops.map_difference import MapDifference, difference_weight

        c = self.config
        vecs = [getattr(self, n) for n in self.difference_names]
        if torch.is_grad_enabled():
            return MapDifference(difference_weight(*vecs, c.differential), 1.0 - c.differential, c.norm_eps)
        key = tuple((p.data_ptr(), p._version, p.dtype) for p in vecs)
        if self._difference is None or self._difference[0] != key:
            self._difference = (key, MapDifference(difference_weight(*(p.detach() for p in vecs), c.differential), 1.0 - c.differential, c.norm_eps))
        return self._difference[1]

    def train(self, mode: bool = True):
        if self.config.differential is not None:
            self._difference = None
        return super().train(mode)

    def _temper_and_mix(self, q, v, v_first):
        """Differentiable forms of the head temperatures and of value mixing."""
        if self.config.head_temperature:
            q = (q.float() * self.temperature.float()[:, None]).to(q.dtype)
        if self.config.value_mixing and v_first is not None:
            from ..ops.qkv_prep import mix_values

            v = mix_values(v, v_first, self.value_mix)
        return q, v

    def forward(self, x: torch.Tensor, mask: Union[None, AttentionMask, torch.Tensor] = None,
                pos_ids: Optional[torch.Tensor] = None, *, skip_out_bias: bool = False,
                residual: Optional[torch.Tensor] = None, row_parallel=None, v_first: Optional[torch.Tensor] = None) -> torch.Tensor:
        """``row_parallel``: a ``TensorParallel`` whose ``row_linear`` applies the output projection and sums it over the model
        axis (the caller then adds the bias once).  ``v_first``: see :meth:`forward_mixing_values`."""
        return self._forward(x, mask, pos_ids, skip_out_bias, residual, row_parallel, v_first)[0]

    def forward_mixing_values(self, x, mask=None, pos_ids=None, v_first: Optional[torch.Tensor] = None):
        """``(attention(x), v_first)`` for layers whose values are mixed with those of the first such layer: that layer is given None and
        returns its own values, the others return what they were given."""
        return self._forward(x, mask, pos_ids, False, None, None, v_first)

    def _forward(self, x, mask, pos_ids, skip_out_bias, residual, row_parallel, v_first):
        c = self.config
        q, k, v = self._compute_qkv(x, pos_ids)
        q, v = self._temper_and_mix(q, v, v_first)
        first = v if v_first is None and c.value_mixing else v_first
        if c.sliding_window is not None and isinstance(mask, AttentionMask) and mask.is_causal:
            mask = mask & AttentionMask.causal(sliding_window=c.sliding_window)
        if c.attention_chunk_size is not None:
            mask = (mask if isinstance(mask, AttentionMask) else AttentionMask.explicit(mask) if mask is not None
                    else AttentionMask.causal()).with_chunk_size(c.attention_chunk_size)
        squeeze = q.dim() == 3
        if squeeze:
            q, k, v = q.unsqueeze(0), k.unsqueeze(0), v.unsqueeze(0)
        maps = [dot_product_attention(
            q[:, :, i::c.maps], k[:, :, i::c.maps], v, mask, attention_dtype=torch.float32 if c.upcast_attn else None, attn_backend=c.attn_backend,
            flash_block_size=c.flash_attention_block_size, logits_soft_cap=c.logits_soft_cap,
            scaling_factor=c.scaling_factor, inference=True) for i in range(c.maps)]
        attn = maps[0]
        if c.differential is not None:
            attn = self.map_difference()(*maps)
        if squeeze:
            attn = attn.squeeze(0)
        if c.head_gate:
            attn = attn.float() * torch.sigmoid(self.g_proj(x).float()).unsqueeze(-1)
        attn = attn.reshape(*x.shape[:-1], self.local_heads * c.v_head_size).to(x.dtype)
        if c.output_gate:
            attn = attn * torch.sigmoid(self.g_proj(x).float()).to(attn.dtype)
        if residual is not None:
            if type(self.o_proj) is Linear:
                from ..ops.gemm import linear_residual

                return linear_residual(attn, self.o_proj.weight, None if skip_out_bias else self.o_proj.bias, residual), first
            return self.o_proj(attn, skip_bias=skip_out_bias) + residual, first  # wrapped projections (LoRA, fp8) add it themselves
        if row_parallel is not None:
            return row_parallel.row_linear(attn, self.o_proj), first
        return self.o_proj(attn, skip_bias=skip_out_bias), first

    def forward_with_residual(self, x, mask, pos_ids, residual):
        """``residual + attention(x)`` with the add done in the output-projection GEMM epilogue."""
        return self.forward(x, mask, pos_ids, residual=residual)

    def paged_decode(self, x: torch.Tensor, kv_cache: "KvPageCache", batch_info, pos_ids: torch.Tensor,
                     residual: Optional[torch.Tensor] = None):
        """Decode/prefill step over packed tokens ``x[T, E]``; writes K/V into the page cache and attends over
        the pages of each sequence (src/levanter/layers/attention.py:1559-1604)."""
        from ..ops import paged_attention as PA

        c = self.config
        if c.output_gate or c.attention_chunk_size is not None or c.v_head_size != c.head_size or c.sliding_window is not None \
                or c.head_temperature or c.value_mixing or c.head_gate or c.differential is not None or (self.rot is not None and not self.rot.is_plain):
            out, _ = self._paged_heads(x, kv_cache, batch_info, pos_ids)
            return (self.o_proj(out) if residual is None else self.o_proj(out) + residual), kv_cache
        q, k, v = self._compute_qkv(x, pos_ids)
        kv_cache = kv_cache.update(batch_info, k, v)
        scale = c.scaling_factor if c.scaling_factor is not None else 1.0 / math.sqrt(c.head_size)
        seg = getattr(batch_info, "prefill_segment_ids", None)
        if seg is not None and x.is_cuda:
            # pure prefill: nothing to read from the cache, so this is causal attention over the packed tokens with one segment
            # per sequence (the flash kernel), instead of the decode kernel walking pages
            m = AttentionMask.causal(sliding_window=c.sliding_window).with_segment_ids(seg.unsqueeze(0), sorted=True)
            out = dot_product_attention(q.unsqueeze(0), k.unsqueeze(0), v.unsqueeze(0), m, attn_backend=c.attn_backend,
                                        logits_soft_cap=c.logits_soft_cap, scaling_factor=c.scaling_factor, inference=True).squeeze(0)
        else:
            out = PA.ragged_paged_attention(q, kv_cache.kv_pages, batch_info.seq_lens, batch_info.page_indices,
                                            batch_info.cu_q_lens, batch_info.num_seqs, sm_scale=scale,
                                            soft_cap=c.logits_soft_cap)
        out = out.reshape(x.shape[0], self.local_heads * c.head_size).to(x.dtype)
        if residual is not None:
            if type(self.o_proj) is Linear:
                from ..ops.gemm import linear_residual

                return linear_residual(out, self.o_proj.weight, self.o_proj.bias, residual), kv_cache
            return self.o_proj(out) + residual, kv_cache
        return self.o_proj(out), kv_cache

    def _fused_projection(self):
        """``(weight, bias or None)`` of the joint projection ``[q; k; v; gate]`` for serving: the projections read the same rows, so a
        decode step streams one matrix instead of launching four products.  None when a projection is wrapped (LoRA, fp8) or only
        some of q, k, v have a bias, and for a model in training.  (The gate per head has none: its rows of the bias are zeros.)"""
        mods = self._projections()
        if self.training or not all(type(m) is Linear for m in mods):
            return None
        with_bias = mods[:3] if self.config.head_gate else mods
        biased = [m.bias is not None for m in with_bias]
        if any(biased) != all(biased):
            return None
        w = self._rows.get([m.weight for m in mods])
        b = self._bias_rows.get([m.bias for m in with_bias]) if w is not None and biased[0] else None
        return None if w is None or (biased[0] and b is None) else (w, b)

    def _paged_heads(self, x, kv_cache: "KvPageCache", batch_info, pos_ids, v_first: Optional[torch.Tensor] = None):
        """``(heads, v_first)``: the (gated) concatenated heads ``[T, heads * v_head_size]`` of packed tokens, for the forms of attention
        that the plain paged path does not have (chunks, windows, a value size of its own, an output gate, temperatures, mixed values,
        partial rotations), and the values that later layers mix with."""
        from ..ops import flash_attention as FA
        from ..ops import paged_attention as PA
        from ..ops.qkv_prep import prepare_qkv
        from ..ops.residual_stream import project

        c = self.config
        T, D, Dv = x.shape[0], c.head_size, c.v_head_size
        nq, nk, nv = c.maps * self.local_heads * D, c.maps * self.local_kv * D, self.local_kv * Dv
        fused = self._fused_projection() if (x.is_cuda and not torch.is_grad_enabled() and self.q_norm is None) else None
        gate = None
        if fused is not None:
            y = project(x, fused[0], bias=fused[1])
            q, k, v = y[:, :nq].unflatten(1, (-1, D)), y[:, nq:nq + nk].unflatten(1, (-1, D)), y[:, nq + nk:nq + nk + nv].unflatten(1, (-1, Dv))
            if c.output_gate or c.head_gate:
                gate = y[:, nq + nk + nv:nq + nk + nv + self.g_proj.weight.shape[0]]
        else:
            q, k, v = self._compute_qkv(x, pos_ids, rotate=False)
            if c.output_gate or c.head_gate:
                gate = self.g_proj(x)
        if self.rot is not None or c.head_temperature or c.value_mixing:
            q, k, v = prepare_qkv(q, k, v, kv_cache.kv_pages, batch_info.new_token_dests, pos_ids, rot=self.rot,
                                  head_scale=self.temperature if c.head_temperature else None, v_first=v_first if c.value_mixing else None,
                                  mix=self.value_mix if c.value_mixing else None)
            if c.value_mixing and v_first is None:
                v_first = v
        else:
            PA.kv_page_write_general(kv_cache.kv_pages, k, v, batch_info.new_token_dests)
        scale = c.scaling_factor if c.scaling_factor is not None else 1.0 / math.sqrt(D)
        seg = getattr(batch_info, "prefill_segment_ids", None)
        kw = dict(chunk=c.attention_chunk_size, window=c.sliding_window, gate=gate, difference=None if c.differential is None else self.map_difference())
        if seg is not None and FA.packed_supported(q, k, v, scale, c.maps):
            # pure prefill: every sequence starts at position 0, nothing is read back from the cache
            out = FA.flash_attention_packed(q, k, v, pos_ids, scaling_factor=scale, logits_soft_cap=c.logits_soft_cap, **kw)
        else:
            out = PA.paged_attention_general(q, kv_cache.kv_pages, self.local_kv, Dv, batch_info, sm_scale=scale, soft_cap=c.logits_soft_cap, **kw)
        return out.reshape(T, self.local_heads * Dv).to(x.dtype), v_first

    def paged_decode_stream(self, x: torch.Tensor, kv_cache: "KvPageCache", batch_info, pos_ids, stream: torch.Tensor):
        """:meth:`paged_decode` for an fp32 residual stream: ``stream + o_proj(heads)``, added in the projection's epilogue."""
        from ..ops.residual_stream import add_linear

        out, _ = self._paged_heads(x, kv_cache, batch_info, pos_ids)
        if type(self.o_proj) is Linear and self.o_proj.bias is None:
            return add_linear(stream, out, self.o_proj.weight), kv_cache
        return stream + self.o_proj(out).float(), kv_cache

    def paged_decode_mixing_values(self, x: torch.Tensor, kv_cache: "KvPageCache", batch_info, pos_ids, v_first: Optional[torch.Tensor] = None):
        """:meth:`paged_decode` of a block whose output is normed before it joins the stream: ``(o_proj(heads) in fp32, v_first)``, with
        ``v_first`` as in :meth:`forward_mixing_values`."""
        from ..ops.residual_stream import project

        out, v_first = self._paged_heads(x, kv_cache, batch_info, pos_ids, v_first)
        if type(self.o_proj) is Linear:
            return project(out, self.o_proj.weight, bias=self.o_proj.bias, out_dtype=torch.float32), v_first
        return self.o_proj(out).float(), v_first

    def empty_page_cache(self, max_pages: int, page_size: int, *, dtype=torch.bfloat16, device=None) -> "KvPageCache":
        c = self.config
        return KvPageCache.init(max_pages, page_size, self.local_kv, c.maps * c.head_size, v_head_size=c.v_head_size, dtype=dtype, device=device)


class AttentionWithSink(Attention):
    """Attention with learned sink logits ``sinks[kv_head, q_heads_per_group]``
    (src/levanter/layers/attention.py:2216-2295)."""

    def __init__(self, config: AttentionConfig, **kw):
        super().__init__(config, **kw)
        self.sinks = nn.Parameter(torch.zeros(self.local_kv, config.q_heads_per_group))
        self.sinks.lev_shape = tuple(self.sinks.shape)

    def forward(self, x, mask=None, pos_ids=None):
        c = self.config
        q, k, v = self._compute_qkv(x, pos_ids)
        squeeze = q.dim() == 3
        if squeeze:
            q, k, v = q.unsqueeze(0), k.unsqueeze(0), v.unsqueeze(0)
        attn = dot_product_attention_with_sink(q, k, v, self.sinks.reshape(-1), mask,
                                               attention_dtype=torch.float32 if c.upcast_attn else None,
                                               logits_soft_cap=c.logits_soft_cap, scaling_factor=c.scaling_factor)
        if squeeze:
            attn = attn.squeeze(0)
        return self.o_proj(attn.reshape(*x.shape[:-1], -1).to(x.dtype))


# --------------------------------------------------------------------------------------------- MLA
@dataclass(frozen=True)
class MultiHeadLatentAttentionConfig:
    """DeepSeek-V3-style latent attention (src/levanter/layers/attention.py:1994-2060)."""

    hidden_dim: int
    num_heads: int
    kv_lora_rank: int
    q_lora_rank: Optional[int] = None
    qk_rope_head_dim: int = 64
    qk_nope_head_dim: int = 128
    v_head_dim: int = 128
    use_bias: bool = False
    upcast_attn: bool = False
    attn_backend: Optional[AttentionBackend] = None
    flash_attention_block_size: Optional[int] = None
    rope: Optional[RotaryEmbeddingsConfig] = None
    scaling_factor: Optional[float] = None
    logits_soft_cap: Optional[float] = None
    norm_eps: float = 1e-6
    sliding_window: Optional[int] = None  # a query sees itself and that many positions less one before it
    sink: bool = False  # a learned number per head joins the softmax denominator (unscaled, with no key and no value)
    output_gate: bool = False  # the heads are multiplied by sigmoid(W_g x) before the output projection
    shares_latent: bool = False  # no down projection of its own: keys and values come from the latents that an earlier layer keeps

    @property
    def softmax_scale(self) -> float:
        return self.scaling_factor if self.scaling_factor is not None else 1.0 / math.sqrt(self.qk_head_dim)

    @property
    def qk_head_dim(self):
        return self.qk_nope_head_dim + self.qk_rope_head_dim


class MultiHeadLatentAttention(nn.Module):
    """K/V are reconstructed from a low-rank latent (``kv_lora_rank``) plus a decoupled RoPE key shared by all heads (none with
    ``qk_rope_head_dim`` 0: attention without positions);
    queries optionally pass through their own low-rank bottleneck (src/levanter/layers/attention.py:2063-2213).

    Serving (:meth:`paged_decode`) caches the normed latent and the rotated key part of a token, ``kv_lora_rank + qk_rope_head_dim``
    numbers for all heads.  Prompts that start in a step are attended to with per-head keys and values: one product of the cache
    rows with ``[[W_uk, 0], [0, 1]]`` yields whole keys, the identity block putting the shared part into every head.  Otherwise
    (decoding, portions) ``W_uk`` is applied to the queries and ``W_uv`` to the result, and the heads read the cache rows as they are.

    With ``shares_latent`` a layer is handed what an earlier layer of the same latent size and rotation keeps: its pages and, for prompts that
    start in a step, its rows of the step."""

    def __init__(self, config: MultiHeadLatentAttentionConfig, init_std: float = 0.02):
        super().__init__()
        c = config
        self.config = c
        H = c.num_heads
        if c.q_lora_rank is None:
            self.q_proj = Linear(c.hidden_dim, H * c.qk_head_dim, bias=c.use_bias, init_std=init_std)
            self.q_a_proj = self.q_a_norm = self.q_b_proj = None
        else:
            self.q_proj = None
            self.q_a_proj = Linear(c.hidden_dim, c.q_lora_rank, bias=c.use_bias, init_std=init_std)
            self.q_a_norm = RmsNorm(c.q_lora_rank, eps=c.norm_eps)
            self.q_b_proj = Linear(c.q_lora_rank, H * c.qk_head_dim, bias=c.use_bias, init_std=init_std)
        self.kv_a_proj = self.kv_a_norm = None
        if not c.shares_latent:
            self.kv_a_proj = Linear(c.hidden_dim, c.kv_lora_rank + c.qk_rope_head_dim, bias=c.use_bias, init_std=init_std)
            self.kv_a_norm = RmsNorm(c.kv_lora_rank, eps=c.norm_eps)
        self.g_proj = Linear(c.hidden_dim, H * c.v_head_dim, init_std=init_std) if c.output_gate else None
        self.kv_b_proj = Linear(c.kv_lora_rank, H * (c.qk_nope_head_dim + c.v_head_dim), bias=c.use_bias, init_std=init_std)
        self.o_proj = Linear(H * c.v_head_dim, c.hidden_dim, bias=c.use_bias, init_std=init_std)
        rope = c.rope if c.rope is not None else DefaultRotaryEmbeddingsConfig()
        self.rot = rope.build(c.qk_rope_head_dim) if c.qk_rope_head_dim > 0 else None
        if c.sink:
            self.sinks = nn.Parameter(torch.zeros(H))
            self.sinks.lev_shape = (H,)
        self._rows, self._whole_kv, self._sinks = FusedRows(-sum(m.weight.shape[0] for m in self._from_input()) % 8), None, None

    def _from_input(self):
        """The projections that read the layer's input."""
        return [m for m in (self.q_proj, self.q_a_proj, self.kv_a_proj, self.g_proj) if m is not None]

    def sinks_fp32(self) -> Optional[torch.Tensor]:
        """The sink numbers in fp32 at a fixed address (it goes into captured graphs), made again like :meth:`_whole_kv_weight`."""
        if not self.config.sink:
            return None
        s = self.sinks
        key = (s.data_ptr(), s._version, s.dtype, s.device)
        if self._sinks is None or self._sinks[0] != key:
            self._sinks = (key, s.detach().float().contiguous().clone())
        return self._sinks[1]

    def up_projections(self, weight: torch.Tensor):
        """``(W_uk [H, qk_nope_head_dim, rank], W_uv [H, v_head_dim, rank])``: views of ``kv_b_proj``'s weight (or of its gradient and the
        like)."""
        c = self.config
        w = weight.view(c.num_heads, c.qk_nope_head_dim + c.v_head_dim, c.kv_lora_rank)
        return w[:, :c.qk_nope_head_dim], w[:, c.qk_nope_head_dim:]

    def _whole_kv_weight(self) -> torch.Tensor:
        """``[H * qk_head_dim + H * v_head_dim, rank + rope]``: rows that turn ``[c, k_rot]`` into every head's key and then every head's
        value.  Derived from ``kv_b_proj``; made again when its weight has moved or changed, and after every change of mode (an optimizer
        writes into flat buffers behind the parameters)."""
        c = self.config
        w = self.kv_b_proj.weight
        key = (w.data_ptr(), w._version, w.dtype, w.device)
        if self._whole_kv is None or self._whole_kv[0] != key:
            H, r, rank = c.num_heads, c.qk_rope_head_dim, c.kv_lora_rank
            uk, uv = self.up_projections(w.detach())
            keys = w.new_zeros(H, c.qk_head_dim, rank + r)
            keys[:, :c.qk_nope_head_dim, :rank] = uk
            keys[:, c.qk_nope_head_dim:, rank:] = torch.eye(r, dtype=w.dtype, device=w.device)
            values = w.new_zeros(H, c.v_head_dim, rank + r)
            values[..., :rank] = uv
            self._whole_kv = (key, torch.cat([keys.flatten(0, 1), values.flatten(0, 1)]))
        return self._whole_kv[1]

    def train(self, mode: bool = True):
        self._whole_kv = self._sinks = None
        return super().train(mode)

    def empty_page_cache(self, max_pages: int, page_size: int, *, dtype=torch.bfloat16, device=None) -> "KvPageCache":
        c = self.config
        return KvPageCache.init(max_pages, page_size, 1, c.kv_lora_rank + c.qk_rope_head_dim, v_head_size=0, dtype=dtype, device=device)

    def paged_decode(self, x: torch.Tensor, kv_cache: "KvPageCache", batch_info, pos_ids: torch.Tensor) -> torch.Tensor:
        """Packed rows ``x [T, hidden]`` of a serving step -> ``[T, hidden]`` in fp32; their latents enter the cache."""
        from ..ops.residual_stream import project

        heads, _ = self._paged_heads(x, kv_cache, batch_info, pos_ids)
        if type(self.o_proj) is Linear:
            return project(heads, self.o_proj.weight, out_dtype=torch.float32)
        return self.o_proj(heads).float()

    def paged_decode_stream(self, x: torch.Tensor, kv_cache: "KvPageCache", batch_info, pos_ids, stream: torch.Tensor):
        """:meth:`paged_decode` for an fp32 residual stream: ``stream + o_proj(heads)``, added in the projection's epilogue."""
        return self.paged_decode_stream_sharing(x, kv_cache, batch_info, pos_ids, stream)[0], kv_cache

    def paged_decode_stream_sharing(self, x: torch.Tensor, kv_cache: "KvPageCache", batch_info, pos_ids, stream: torch.Tensor,
                                    latent: Optional[torch.Tensor] = None):
        """``(stream + o_proj(heads), latent)`` for layers of which some read what others keep.  ``latent [T, rank + rope]``: the rows of the
        step that entered the cache, where a layer had use for them (None otherwise, and then they are read from the cache); a layer that
        shares them is given them, with the pages of the layer that keeps them."""
        from ..ops.residual_stream import add_linear

        heads, latent = self._paged_heads(x, kv_cache, batch_info, pos_ids, latent)
        if type(self.o_proj) is Linear and self.o_proj.bias is None:
            return add_linear(stream, heads, self.o_proj.weight), latent
        return stream + self.o_proj(heads).float(), latent

    def _paged_heads(self, x: torch.Tensor, kv_cache: "KvPageCache", batch_info, pos_ids: torch.Tensor, latent: Optional[torch.Tensor] = None):
        """``(heads, latent)``: the concatenated (gated) heads ``[T, heads * v_head_dim]`` of packed rows; ``latent`` as in
        :meth:`paged_decode_stream_sharing`."""
        from ..ops import flash_attention as FA
        from ..ops import paged_attention as PA
        from ..ops.qkv_prep import norm_rows, prepare_latent, rotate_queries
        from ..ops.residual_stream import project

        c = self.config
        if c.logits_soft_cap is not None or c.use_bias:
            raise NotImplementedError("serving latent attention takes neither a soft cap nor biases")
        T, H, dn, dr, dv, rank = x.shape[0], c.num_heads, c.qk_nope_head_dim, c.qk_rope_head_dim, c.v_head_dim, c.kv_lora_rank
        nq = H * c.qk_head_dim
        mods = self._from_input()
        w = None
        if all(type(m) is Linear for m in mods) and x.is_cuda and not self.training and not torch.is_grad_enabled():
            w = self._rows.get([m.weight for m in mods])
        if w is not None:
            parts = project(x, w).split([m.weight.shape[0] for m in mods] + [self._rows.pad], dim=1)
        else:
            parts = [m(x) for m in mods]
        q, rest = parts[0], list(parts[1:])
        down = rest.pop(0) if self.kv_a_proj is not None else None
        gate = rest.pop(0) if self.g_proj is not None else None
        if self.q_a_proj is not None:
            q = norm_rows(q, self.q_a_norm.weight, self.q_a_norm.eps)
            q = project(q, self.q_b_proj.weight) if type(self.q_b_proj) is Linear else self.q_b_proj(q)
        q = q.unflatten(1, (H, c.qk_head_dim))
        pages, dests = kv_cache.kv_pages, batch_info.new_token_dests
        weight, sink = self.kv_b_proj.weight, self.sinks_fp32()

        def prepare(q_out, to_cache_only):
            """Rotated queries (into ``q_out``, or in place) and, unless another layer has seen to it, the latents in the cache."""
            if c.shares_latent:
                if self.rot is not None:
                    rotate_queries(q[..., dn:], pos_ids, self.rot, q_out)
                return latent
            return prepare_latent(down, self.kv_a_norm.weight, self.kv_a_norm.eps, pages, dests, pos_ids, self.rot, q[..., dn:], q_out,
                                  to_cache_only=to_cache_only)[0]

        if getattr(batch_info, "prefill_segment_ids", None) is not None and self._packed_prefill_fits(q) and (latent is not None or not c.shares_latent):
            latent = prepare(None, False)
            kv = project(latent, self._whole_kv_weight())
            k, v = kv[:, :nq].unflatten(1, (H, c.qk_head_dim)), kv[:, nq:].unflatten(1, (H, dv))
            heads = FA.flash_attention_packed(q, k, v, pos_ids, scaling_factor=c.softmax_scale, window=c.sliding_window, sink=sink, gate=gate)
        else:
            uk, uv = self.up_projections(weight)
            qa = q.new_empty(T, H, rank + dr)
            latent = prepare(qa[..., rank:], True)
            PA.head_product(q[..., :dn], uk.to(q.dtype), qa[..., :rank], b_trans=False)
            o = PA.paged_attention_latent(qa, pages, rank, batch_info, sm_scale=c.softmax_scale, window=c.sliding_window, sink=sink)
            heads = PA.head_product(o.to(q.dtype), uv.to(q.dtype), q.new_empty(T, H, dv), b_trans=True, gate=gate)
        return heads.reshape(T, H * dv).to(x.dtype), latent

    def _packed_prefill_fits(self, q: torch.Tensor) -> bool:
        """Whether the packed flash kernel takes this layer's sizes (the joint product of keys and values has the strides of its columns)."""
        from ..ops.flash_attention import packed_rows_ok

        c = self.config
        return (packed_rows_ok(q, 192) and q.shape[0] % 256 == 0 and c.softmax_scale > 0.0 and c.v_head_dim % 8 == 0 and c.v_head_dim <= 128
                and (c.kv_lora_rank + c.qk_rope_head_dim) % 8 == 0 and type(self.kv_b_proj) is Linear and self.kv_b_proj.weight.dtype == q.dtype
                and not torch.is_grad_enabled())

    def forward(self, x, mask=None, pos_ids=None):
        return self.forward_sharing(x, mask, pos_ids)[0]

    def forward_sharing(self, x, mask=None, pos_ids=None, kept=None):
        """``(attention(x), kept)`` for layers of which some read what others keep: ``kept`` is ``(latent [B, S, rank], rotated key part)``, made
        here unless the layer shares an earlier one's."""
        c = self.config
        if c.sliding_window is not None:
            mask = (mask if isinstance(mask, AttentionMask) else AttentionMask.explicit(mask) if mask is not None
                    else AttentionMask.causal()) & AttentionMask.causal(sliding_window=c.sliding_window)
        B, S, _ = x.shape
        H = c.num_heads
        if pos_ids is None:
            pos_ids = torch.arange(S, device=x.device)
        q = self.q_proj(x) if self.q_proj is not None else self.q_b_proj(self.q_a_norm(self.q_a_proj(x)))
        q = q.view(B, S, H, c.qk_head_dim)
        q_nope, q_rope = q.split([c.qk_nope_head_dim, c.qk_rope_head_dim], dim=-1)
        if not c.shares_latent:
            latent, k_rope = self.kv_a_proj(x).split([c.kv_lora_rank, c.qk_rope_head_dim], dim=-1)
            kept = (self.kv_a_norm(latent), k_rope if self.rot is None else self.rot(k_rope.unsqueeze(2), pos_ids).squeeze(2))
        latent, k_rope = kept
        kv = self.kv_b_proj(latent).view(B, S, H, c.qk_nope_head_dim + c.v_head_dim)
        k_nope, v = kv.split([c.qk_nope_head_dim, c.v_head_dim], dim=-1)
        qf, kf = q_nope, k_nope
        if self.rot is not None:
            qf = torch.cat([q_nope, self.rot(q_rope, pos_ids)], dim=-1)
            kf = torch.cat([k_nope, k_rope.unsqueeze(2).expand(B, S, H, c.qk_rope_head_dim)], dim=-1)
        scale = c.softmax_scale

        def project_out(heads):
            heads = heads.reshape(B, S, H * c.v_head_dim)
            if self.g_proj is not None:
                heads = heads.float() * torch.sigmoid(self.g_proj(x).float())
            return self.o_proj(heads.to(x.dtype))

        if c.sink:
            if c.logits_soft_cap is not None:
                raise NotImplementedError("latent attention with a sink takes no soft cap")
            # the sink is a key column of its own whose value row is zero
            s = torch.einsum("bqhd,bkhd->bhqk", qf.float() * scale, kf.float())
            m = materialize_mask(mask, S, S, device=x.device)
            if m is not None:
                s = torch.where(m, s, torch.full_like(s, -1e9))
            p = torch.softmax(torch.cat([s, self.sinks.float().view(1, H, 1, 1).expand(B, H, S, 1)], dim=-1), dim=-1)[..., :-1]
            return project_out(torch.einsum("bhqk,bkhd->bqhd", p.to(v.dtype), v)), kept
        # value head size differs from the qk head size, so pad V for the shared kernel interface
        out = simple_attention_with_dropout(qf, kf, F.pad(v, (0, c.qk_head_dim - c.v_head_dim)) if c.v_head_dim < c.qk_head_dim else v,
                                            mask, attention_dtype=torch.float32 if c.upcast_attn else None,
                                            logits_soft_cap=c.logits_soft_cap, scaling_factor=scale)
        return project_out(out[..., : c.v_head_dim]), kept


# --------------------------------------------------------------------------------------------- paged KV cache
@dataclass
class KvPageCache:
    """Paged KV storage ``kv_pages[page, slot, 2 * kv_heads, head_size]`` with K at even and V at odd head index
    (src/levanter/layers/attention.py:1638-1707); with a value size of its own ``kv_pages[page, slot, kv_heads, head_size + v_head_size]``,
    the same order in memory: per KV head a key row, then a value row.  Latent attention keeps one row for all heads, whose first
    part is also the value (``v_head_size`` 0)."""

    kv_pages: torch.Tensor

    @staticmethod
    def init(max_pages: int, page_size: int, kv_heads: int, head_size: int, *, v_head_size: Optional[int] = None, dtype=torch.bfloat16,
             device=None):
        if v_head_size is not None and v_head_size != head_size:
            return KvPageCache(torch.zeros(max_pages, page_size, kv_heads, head_size + v_head_size, dtype=dtype, device=device))
        return KvPageCache(torch.zeros(max_pages, page_size, 2 * kv_heads, head_size, dtype=dtype, device=device))

    @property
    def page_size(self) -> int:
        return self.kv_pages.shape[1]

    def update(self, batch_info, new_k: torch.Tensor, new_v: torch.Tensor) -> "KvPageCache":
        """Scatter ``new_k/new_v [T, kv_heads, D]`` to the (page, slot) destinations of ``batch_info``;
        destinations outside the table (padding tokens) are dropped."""
        from ..ops import paged_attention as PA

        PA.kv_page_write(self.kv_pages, new_k, new_v, batch_info.new_token_dests)
        return self

    def copy_page(self, src_page: int, dst_page: int) -> "KvPageCache":
        self.kv_pages[dst_page].copy_(self.kv_pages[src_page])
        return self

    def copy_slot(self, src: int, dst: int) -> "KvPageCache":
        return self  # nothing is kept by slots


def default_ragged_paged_attention(q, kv_pages, kv_lens, page_indices, cu_q_lens, num_seqs, sm_scale: float = 1.0, soft_cap=None):
    """The plain statement of ragged paged attention (src/levanter/layers/attention.py:1856-1991): per sequence, causal by
    absolute position over the pages it owns.  The engine calls ``ops.paged_attention.ragged_paged_attention`` (the CUDA kernel
    on a B200); this is its oracle under the reference's name."""
    from ..ops.paged_attention import ragged_paged_attention_reference

    return ragged_paged_attention_reference(q, kv_pages, kv_lens, page_indices, cu_q_lens, num_seqs, sm_scale, soft_cap)
