"""Recurrent token mixers that serve beside attention: the layer, and the state that a sequence keeps instead of keys and values."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Optional, Tuple

import torch
import torch.nn as nn

from ..nn import FusedRows, Linear, RmsNorm
from ..ops.gated_scan import min_gru, min_gru_packed
from ..ops.linear_attention import fixed_decay_attention, gated_norm, linear_attention_packed
from ..ops.residual_stream import add_linear, project
from .attention import AttentionMask


@dataclass
class SlotStateCache:
    """Fixed-size recurrent state ``state[slot, ...]`` (fp32) per sequence slot of the page table.  A slot that is taken again needs no
    reset: the layers start a sequence from zero at its position 0."""

    state: torch.Tensor

    @staticmethod
    def init(max_seqs: int, *size: int, device=None) -> "SlotStateCache":
        return SlotStateCache(torch.zeros(max_seqs, *size, dtype=torch.float32, device=device))

    def copy_slot(self, src: int, dst: int) -> "SlotStateCache":
        self.state[dst].copy_(self.state[src])
        return self

    def copy_page(self, src_page: int, dst_page: int) -> "SlotStateCache":
        return self  # nothing is kept by pages


def sequence_starts(mask) -> Optional[torch.Tensor]:
    """``[B, L]`` bool: where packed sequences (segment ids of the mask) begin; None when rows are whole sequences."""
    if not isinstance(mask, AttentionMask) or mask.segment_ids is None:
        return None
    seg = _segments(mask)
    starts = torch.ones_like(seg, dtype=torch.bool)
    starts[:, 1:] = seg[:, 1:] != seg[:, :-1]
    return starts


def _segments(mask: AttentionMask) -> torch.Tensor:
    seg = mask.segment_ids[0]
    return seg if seg.dim() == 2 else seg[None]


class MinGru(nn.Module):
    """minGRU: ``o_proj(S_t * silu(g_proj x))`` over ``S_t = (1 - z) S_{t-1} + z c`` whose gates read the current token only: ``z =
    sigmoid(z_proj x)``, ``c = u + 1/2`` for ``u = x_proj x >= 0`` and ``sigmoid(u)`` below."""

    def __init__(self, hidden_dim: int, width: int, *, init_std: float = 0.02):
        super().__init__()
        self.width = width
        self.z_proj = Linear(hidden_dim, width, bias=True, init_std=init_std)
        self.x_proj = Linear(hidden_dim, width, bias=True, init_std=init_std)
        self.g_proj = Linear(hidden_dim, width, init_std=init_std)
        self.o_proj = Linear(width, hidden_dim, init_std=init_std)
        self._rows, self._bias = FusedRows(), FusedRows(pad=width)  # the output gate has no bias

    def _gated(self, states: torch.Tensor, g: torch.Tensor, dtype) -> torch.Tensor:
        return (states * torch.nn.functional.silu(g.float())).to(dtype)

    def forward(self, x: torch.Tensor, mask=None, pos_ids=None) -> torch.Tensor:
        """``x [B, L, hidden]`` (or ``[L, hidden]``); packed sequences (segment ids of the mask) start from zero each."""
        starts = sequence_starts(mask)
        z, u, g = self.z_proj(x), self.x_proj(x), self.g_proj(x)
        z3, u3 = (z, u) if z.dim() == 3 else (z[None], u[None])
        s = min_gru(z3, u3, starts)
        return self.o_proj(self._gated(s if z.dim() == 3 else s[0], g, x.dtype))

    def paged_decode(self, x: torch.Tensor, cache: SlotStateCache, batch_info, pos_ids=None) -> torch.Tensor:
        """Packed rows ``x [T, hidden]`` of a serving step -> ``[T, hidden]`` in fp32; the sequences' states go on from their slots."""
        mods = (self.z_proj, self.x_proj, self.g_proj)
        plain = all(type(m) is Linear for m in mods) and not self.training and not torch.is_grad_enabled()
        w = self._rows.get([m.weight for m in mods]) if plain else None
        b = self._bias.get([self.z_proj.bias, self.x_proj.bias]) if w is not None else None
        if w is not None and b is not None:
            y = project(x, w, bias=b, out_dtype=torch.float32)
        else:
            y = torch.cat([m(x).float() for m in mods], dim=1)
        h = min_gru_packed(y, cache.state, batch_info, x.dtype)
        if type(self.o_proj) is Linear:
            return project(h, self.o_proj.weight, out_dtype=torch.float32)
        return self.o_proj(h).float()

    def empty_state(self, max_seqs: int, device=None) -> SlotStateCache:
        return SlotStateCache.init(max_seqs, self.width, device=device)


@dataclass(frozen=True)
class LinearAttentionConfig:
    """Linear attention with a fixed decay per head (:class:`LinearAttention`)."""

    hidden_dim: int
    num_heads: int
    head_dim: int
    v_head_dim: int
    decay: Tuple[float, ...]
    key_scale: float = 1.0
    silu: bool = False          # q, k and v pass through silu
    norm_per_head: bool = True  # the heads' outputs are normed one by one without a weight; else all together with one
    sigmoid_gate: bool = False  # the gate is a sigmoid; else a silu
    norm_eps: float = 1e-6

    def __post_init__(self):
        if len(self.decay) != self.num_heads:
            raise ValueError(f"{len(self.decay)} decays for {self.num_heads} heads")


class LinearAttention(nn.Module):
    """``o_proj(norm(o) * act(g_proj x))`` with, per head, ``S_t = decay S_{t-1} + key_scale k_t v_t^T`` and ``o_t = S_t^T q_t`` of q, k, v projected from
    ``x``: retention (Sun et al., "Retentive Network", 2023; ``key_scale = head_dim^-1/2``, norm per head, silu gate) or lightning attention (silu
    on q, k and v, one norm with a weight, sigmoid gate)."""

    def __init__(self, config: LinearAttentionConfig, *, init_std: float = 0.02):
        super().__init__()
        c = self.config = config
        qk, v = c.num_heads * c.head_dim, c.num_heads * c.v_head_dim
        self.q_proj = Linear(c.hidden_dim, qk, init_std=init_std)
        self.k_proj = Linear(c.hidden_dim, qk, init_std=init_std)
        self.v_proj = Linear(c.hidden_dim, v, init_std=init_std)
        self.g_proj = Linear(c.hidden_dim, v, init_std=init_std)
        self.o_proj = Linear(v, c.hidden_dim, init_std=init_std)
        self.o_norm = None if c.norm_per_head else RmsNorm(v, eps=c.norm_eps)
        self._rows = FusedRows(-(2 * qk + 2 * v) % 8)
        self._decay: Dict[torch.device, torch.Tensor] = {}

    def decay_on(self, device) -> torch.Tensor:
        """The decays in fp32 (whatever the parameters' type), made once per device."""
        device = torch.device(device)
        if device not in self._decay:
            self._decay[device] = torch.tensor(self.config.decay, dtype=torch.float32, device=device)
        return self._decay[device]

    def _gated(self, o: torch.Tensor, g: torch.Tensor) -> torch.Tensor:
        """``o, g [T, heads * v_head_dim]``."""
        c = self.config
        return gated_norm(o, g, c.norm_eps, groups=c.num_heads if c.norm_per_head else 1, weight=None if self.o_norm is None else self.o_norm.weight,
                          sigmoid=c.sigmoid_gate)

    def forward(self, x: torch.Tensor, mask=None, pos_ids=None) -> torch.Tensor:
        """``x [B, L, hidden]``; packed sequences (segment ids of the mask) start from zero each."""
        c = self.config
        B, L, _ = x.shape
        q, k, v = (m(x).view(B, L, c.num_heads, -1) for m in (self.q_proj, self.k_proj, self.v_proj))
        if c.silu:
            q, k, v = (torch.nn.functional.silu(t.float()) for t in (q, k, v))
        seg = None
        if isinstance(mask, AttentionMask) and mask.segment_ids is not None:
            seg = _segments(mask).expand(B, L)
        o = fixed_decay_attention(q, k.float() * c.key_scale, v, self.decay_on(x.device), seg).reshape(B * L, -1)
        return self.o_proj(self._gated(o, self.g_proj(x).reshape(B * L, -1).float()).to(x.dtype).view(B, L, -1))

    def paged_decode_stream(self, x: torch.Tensor, cache: SlotStateCache, batch_info, pos_ids, stream: torch.Tensor):
        """Packed rows ``x [T, hidden]`` of a serving step: ``stream + o_proj(...)`` on the fp32 stream, added in the projection's epilogue; the
        sequences' states go on from their slots."""
        c = self.config
        mods = (self.q_proj, self.k_proj, self.v_proj, self.g_proj)
        w = None
        if all(type(m) is Linear for m in mods) and x.is_cuda and not self.training and not torch.is_grad_enabled():
            w = self._rows.get([m.weight for m in mods])
        y = project(x, w) if w is not None else torch.cat([m(x) for m in mods], dim=1)
        qk, nv = c.num_heads * c.head_dim, c.num_heads * c.v_head_dim
        q, k, v, g = y[:, :2 * qk + 2 * nv].split([qk, qk, nv, nv], dim=1)
        heads = lambda t: t.unflatten(1, (c.num_heads, -1))  # noqa: E731
        o = linear_attention_packed(heads(q), heads(k), heads(v), self.decay_on(x.device), cache.state, batch_info, key_scale=c.key_scale, silu=c.silu)
        h = self._gated(o.flatten(1), g)
        if type(self.o_proj) is Linear:
            return add_linear(stream, h, self.o_proj.weight), cache
        return stream + self.o_proj(h).float(), cache

    def empty_state(self, max_seqs: int, device=None) -> SlotStateCache:
        c = self.config
        return SlotStateCache.init(max_seqs, c.num_heads, c.head_dim, c.v_head_dim, device=device)
