"""Mixtures of gated experts behind a softmax router that chooses within groups of neighbouring experts, with an optional shared expert."""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn as nn

from ..models.llama import LlamaMlp
from ..nn import FusedRows, Linear, trunc_normal_
from ..ops import moe
from ..ops.glu import GatedActivation
from ..ops.residual_stream import _kernels, add_linear, glu_of_rows, project
from ..utils.activation import ActivationFunctionEnum


class GatedExperts(nn.Module):
    """Expert weights ``gate_up [E, 2 ff, hidden]`` (an expert's gate rows, then its up rows) and ``down [E, hidden, ff]``."""

    def __init__(self, num_experts: int, hidden: int, intermediate: int, init_std: float):
        super().__init__()
        self.gate_up = nn.Parameter(torch.empty(num_experts, 2 * intermediate, hidden))
        self.down = nn.Parameter(torch.empty(num_experts, hidden, intermediate))
        for w in (self.gate_up, self.down):
            if w.device.type != "meta":
                trunc_normal_(w, init_std)
            w.lev_shape = tuple(w.shape)


class GroupedSoftmaxMoe(nn.Module):
    """``top`` of ``num_experts`` gated experts per token, chosen by softmax scores (of logits with ``router_bias`` if asked for) within the
    ``keep`` best of ``groups`` groups of neighbours (a group counts by its best score), weighed by the chosen scores divided by their sum.
    ``shared_intermediate``: a further expert of that size runs for every token, with ``shared_gated`` multiplied by the sigmoid of one number
    per token.  ``activation`` and ``shared_activation``: of the experts and of the shared one.

    Serving: the shared expert's two projections, the router and the number that weighs the shared expert read the same rows, so they are
    one product with fp32 output."""

    def __init__(self, hidden: int, intermediate: int, num_experts: int, top: int, *, groups: int = 1, keep: int = 1,
                 shared_intermediate: Optional[int] = None, shared_gated: bool = True, activation: GatedActivation = ActivationFunctionEnum.silu,
                 shared_activation: GatedActivation = ActivationFunctionEnum.silu, router_bias: bool = False, init_std: float = 0.02):
        super().__init__()
        self.num_experts, self.top, self.groups, self.keep = num_experts, top, groups, keep
        self.shared_intermediate, self.activation = shared_intermediate, activation
        self.router = Linear(hidden, num_experts, bias=router_bias, init_std=init_std)
        self.experts = GatedExperts(num_experts, hidden, intermediate, init_std)
        rows = num_experts
        if shared_intermediate is not None:
            self.shared = LlamaMlp(hidden, shared_intermediate, shared_activation, init_std=init_std)
            self.shared_gate = Linear(hidden, 1, init_std=init_std) if shared_gated else None
            rows += 2 * shared_intermediate + int(shared_gated)
        self._rows = FusedRows(-rows % 8)

    def _joint_weight(self) -> Optional[torch.Tensor]:
        """``[gate; up; router; shared gate; padding]`` (or the router alone); None in training or when a projection is wrapped."""
        mods = [self.router]
        if self.shared_intermediate is not None:
            mods = [self.shared.gate_proj, self.shared.up_proj, self.router] + ([] if self.shared_gate is None else [self.shared_gate])
        if self.training or not all(type(m) is Linear for m in mods) or (self.shared_intermediate is not None and type(self.shared.down_proj) is not Linear):
            return None
        return self._rows.get([m.weight for m in mods])

    def add_to_stream(self, stream: torch.Tensor, h: torch.Tensor, batch_info=None) -> torch.Tensor:
        """``stream + moe(h)``.  ``batch_info``: padding tokens of a packed batch (no cache destination) are sent to no expert."""
        e, E, ff = self.experts, self.num_experts, self.shared_intermediate or 0
        shape = h.shape
        h2 = h.reshape(-1, shape[-1])
        w = self._joint_weight() if _kernels(h2, stream) else None
        if w is not None:
            y = project(h2, w, out_dtype=torch.float32)
            live, limit = (None, 0) if batch_info is None else (batch_info.new_token_dests, batch_info.num_slots)
            routed = moe.route_softmax(y[:, 2 * ff:2 * ff + E], self.top, groups=self.groups, keep=self.keep, bias=self.router.bias, live=live,
                                       live_limit=limit)
            flat = stream.view(-1, shape[-1])
            moe.add_expert_outputs(flat, h2, routed, e.gate_up, e.down, gated=True, act=self.activation)
            if ff:
                a = glu_of_rows(y, ff, self.shared.act, gate_logit=None if self.shared_gate is None else y[:, 2 * ff + E], out_dtype=h2.dtype)
                add_linear(flat, a, self.shared.down_proj.weight)
            return flat.view(shape)
        z = project(h2, self.router.weight, out_dtype=torch.float32) if type(self.router) is Linear else self.router(h2).float()
        # a plain router leaves its bias to the routing, a wrapped one (LoRA) has added it
        idx, weights = moe.route_softmax_reference(z, self.top, self.groups, self.keep, self.router.bias if type(self.router) is Linear else None)
        out = moe.expert_outputs(h2, idx, weights, e.gate_up, e.down, gated=True, act=self.activation)
        if ff:
            shared = self.shared(h2).float()
            out = out + (shared if self.shared_gate is None else torch.sigmoid(self.shared_gate(h2).float()) * shared)
        return stream + out.view(shape)
