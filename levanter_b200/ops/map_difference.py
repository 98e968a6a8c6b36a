"""Differential attention: a head attends with two score maps over the same values, and its output is the difference of the two results,
normed.  The serving kernels (``csrc/flash_attn_fwd2.cu``, ``csrc/paged_attention.cu``) do the combination where the maps' results
are still in registers or tensor memory; this is its statement, the argument they take, and the differentiable form."""
from __future__ import annotations

from dataclasses import dataclass

import torch


def difference_weight(q1: torch.Tensor, k1: torch.Tensor, q2: torch.Tensor, k2: torch.Tensor, constant: float) -> torch.Tensor:
    """``exp(q1 . k1) - exp(q2 . k2) + constant`` in fp32, ``[1]``: what the second map's result is multiplied by."""
    f = [t.float() for t in (q1, k1, q2, k2)]
    return ((f[0] * f[1]).sum().exp() - (f[2] * f[3]).sum().exp() + constant).reshape(1)


@dataclass(frozen=True)
class MapDifference:
    """``o = a1 - weight * a2``, then ``scale * o / sqrt(mean(o^2) + eps)`` over the values of a head."""

    weight: torch.Tensor  # fp32 [1]
    scale: float
    eps: float

    def __call__(self, a1: torch.Tensor, a2: torch.Tensor) -> torch.Tensor:
        """``a1, a2 [..., v_size]`` -> fp32 of that shape."""
        o = a1.float() - self.weight * a2.float()
        return o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + self.eps) * self.scale
