"""Recurrent token mixers that serve beside attention: the layer, and the state that a sequence keeps instead of keys and values."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn as nn

from ..nn import FusedRows, Linear
from ..ops.gated_scan import min_gru, min_gru_packed
from ..ops.residual_stream import project
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
        starts = None
        if isinstance(mask, AttentionMask) and mask.segment_ids is not None:
            seg = mask.segment_ids[0]
            seg = seg if seg.dim() == 2 else seg[None]
            starts = torch.ones_like(seg, dtype=torch.bool)
            starts[:, 1:] = seg[:, 1:] != seg[:, :-1]
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
