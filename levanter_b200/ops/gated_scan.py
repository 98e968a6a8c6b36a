"""The minimal gated recurrence of minGRU layers: ``z = sigmoid(zl)``, ``c = u + 1/2`` for ``u >= 0`` and ``sigmoid(u)`` below,
``S_t = (1 - z) S_{t-1} + z c``, all in fp32 (``csrc/gated_scan.cu``).

:func:`min_gru_packed` is the serving form: packed rows of several sequences with a state per sequence slot.  :func:`min_gru` is the
differentiable form for whole sequences."""
from __future__ import annotations

from typing import Optional

import torch

from . import lib

_f = {}


def _gates(zl: torch.Tensor, u: torch.Tensor):
    """``(1 - z, z c)``: the affine map of a step."""
    zl, u = zl.float(), u.float()
    cand = torch.where(u >= 0, u + 0.5, torch.sigmoid(u.clamp(max=0.0)))
    return torch.sigmoid(-zl), torch.sigmoid(zl) * cand


def min_gru(zl: torch.Tensor, u: torch.Tensor, starts: Optional[torch.Tensor] = None) -> torch.Tensor:
    """States ``[B, L, W]`` (fp32) for ``zl, u [B, L, W]``.  ``starts [B, L]`` bool: positions where a sequence begins (the state is zero
    before them).  Composes the affine maps in ``log2 L`` passes."""
    a, s = _gates(zl, u)
    if starts is not None:
        a = a.masked_fill(starts.unsqueeze(-1), 0.0)
    step, L = 1, zl.shape[1]
    while step < L:
        s = torch.cat([s[:, :step], a[:, step:] * s[:, :-step] + s[:, step:]], dim=1)
        a = torch.cat([a[:, :step], a[:, step:] * a[:, :-step]], dim=1)
        step *= 2
    return s


def min_gru_packed(y: torch.Tensor, state: torch.Tensor, batch_info, out_dtype: torch.dtype) -> torch.Tensor:
    """``y [T, 3 W]`` fp32: the update-gate logits, the candidate inputs and the output-gate inputs ``g`` of packed rows; ``state [slots, W]``
    fp32, updated in place -> ``S * silu(g)`` ``[T, W]``.  A sequence whose first packed row is its position 0 starts from a zero
    state; padding rows come out as zeros."""
    T, W = y.shape[0], state.shape[1]
    b = batch_info
    if not torch.is_grad_enabled() and y.is_cuda and lib.available() and y.dtype == torch.float32 and y.stride(1) == 1 and state.is_contiguous() \
            and out_dtype in (torch.float32, torch.bfloat16):
        c = lib
        if "m" not in _f:
            _f["m"] = lib.fn("lvb_min_gru_scan", [c.c_void_p] * 9 + [c.c_int, c.c_int, c.c_longlong] + [c.c_int] * 4 + [c.c_void_p])
        i32 = lambda t: t.to(device=y.device, dtype=torch.int32).contiguous()  # noqa: E731
        slots, lens, cu, ns = i32(b.slot_ids), i32(b.seq_lens), i32(b.cu_q_lens), i32(b.num_seqs.reshape(1))
        S = slots.shape[0]
        out = torch.empty(T, W, dtype=out_dtype, device=y.device)
        at = y.data_ptr()
        rc = _f["m"](at, at + 4 * W, at + 8 * W, out.data_ptr(), state.data_ptr(), slots.data_ptr(), lens.data_ptr(), cu.data_ptr(), ns.data_ptr(), T, W,
                     y.stride(0), S, state.shape[0], int(out_dtype == torch.float32), int(T > 4 * S), lib.stream_ptr())
        lib.check_rc(rc, "lvb_min_gru_scan")
        return out
    zl, u, g = y.float().split(W, dim=1)
    a, s = _gates(zl, u)
    out = torch.zeros(T, W, dtype=torch.float32, device=y.device)
    cu, lens, slots = b.cu_q_lens.tolist(), b.seq_lens.tolist(), b.slot_ids.tolist()
    for i in range(int(b.num_seqs)):
        r0, r1 = cu[i], cu[i + 1]
        if r1 <= r0 or not 0 <= slots[i] < state.shape[0]:
            continue
        st = state[slots[i]].clone() if lens[i] > r1 - r0 else torch.zeros_like(state[slots[i]])
        for r in range(r0, r1):
            st = a[r] * st + s[r]
            out[r] = st
        state[slots[i]] = st
    return (out * torch.nn.functional.silu(g)).to(out_dtype)
