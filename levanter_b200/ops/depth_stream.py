"""What happens between the blocks of a model that keeps what every layer has made of its fp32 residual stream (``csrc/depth_stream.cu``): a
weighted sum over depth, RMS norms in groups, and the token shift, which mixes a normed row with the one before it in its sequence.

The kernel runs when no gradient is being recorded; the PyTorch statements are the CPU path and the test oracle."""
from __future__ import annotations

from typing import Optional

import torch

from . import lib
from .residual_stream import _kernels

_f = {}


def grouped_rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float, groups: int) -> torch.Tensor:
    """Each of ``groups`` equal consecutive parts of a row of ``x [..., D]`` divided by its root mean square, then times ``weight [D]``; fp32,
    differentiable."""
    parts = x.float().unflatten(-1, (groups, -1))
    return (parts * torch.rsqrt(parts.pow(2).mean(-1, keepdim=True) + eps)).flatten(-2) * weight.float()


def shift_tokens(h: torch.Tensor, mu: torch.Tensor, starts: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``h + (h' - h) * mu`` for ``h [B, L, D]`` with ``h'`` the previous position's ``h``: zeros at position 0 and where ``starts [B, L]``.
    Differentiable."""
    before = torch.nn.functional.pad(h, (0, 0, 1, 0))[:, :-1]
    if starts is not None:
        before = before.masked_fill(starts.unsqueeze(-1), 0.0)
    return h + (before - h) * mu.float()


def norm_of_depths(history: torch.Tensor, weight: torch.Tensor, eps: float, *, groups: int = 1, coef: Optional[torch.Tensor] = None,
                   out: Optional[torch.Tensor] = None, rows: Optional[torch.Tensor] = None, out_dtype: Optional[torch.dtype] = None,
                   shift: Optional[torch.Tensor] = None, state: Optional[torch.Tensor] = None, batch_info=None) -> torch.Tensor:
    """Forward only.  ``history [n, T, D]`` fp32, ``x = sum_j coef[j] history[j]`` (``coef`` None: ``n`` is 1), ``h`` its RMS norm in groups
    (:func:`grouped_rms_norm`) -> ``h`` in ``out_dtype`` (default: the weight's).

    ``out [T, D]``: receives ``x`` (not one of the planes).  ``rows``: these rows only.  ``shift [D]``: the result is ``h + (h' - h) * shift`` over
    packed rows of sequences, where the row before a sequence's first is its slot's row of ``state [slots, D]`` (zeros at position 0), which
    the sequence's last ``h`` then replaces."""
    n, T, D = history.shape
    dt = out_dtype or weight.dtype
    b = batch_info
    small = [t for t in (coef, weight, shift) if t is not None]
    if _kernels(history, weight) and history.dtype == torch.float32 and history[0].is_contiguous() and dt in (torch.float32, torch.bfloat16) \
            and weight.dtype in (torch.float32, torch.bfloat16) and all(t.dtype == weight.dtype and t.is_contiguous() for t in small) \
            and all(t is None or (t.dtype == torch.float32 and t.is_contiguous()) for t in (out, state)):
        c = lib
        if "d" not in _f:
            _f["d"] = lib.fn("lvb_depth_stream", [c.c_void_p, c.c_longlong, c.c_int] + [c.c_void_p] * 5 + [c.c_int] + [c.c_void_p] * 5 + [c.c_int] * 2 +
                             [c.c_void_p] + [c.c_int] * 4 + [c.c_float, c.c_void_p])
        if rows is not None:
            rows = rows.to(torch.int64).contiguous()
            T = rows.numel()
        y = torch.empty(T, D, dtype=dt, device=history.device)
        seqs, S, slots = (0, 0, 0, 0), 0, 0
        if shift is not None:
            i32 = lambda t: t.to(device=y.device, dtype=torch.int32).contiguous()  # noqa: E731
            tables = [i32(t) for t in (b.slot_ids, b.seq_lens, b.cu_q_lens, b.num_seqs.reshape(1))]
            seqs, S, slots = tuple(t.data_ptr() for t in tables), tables[0].shape[0], state.shape[0]
        rc = _f["d"](history.data_ptr(), history.stride(0), n, lib.ptr(coef), lib.ptr(out), lib.ptr(rows), weight.data_ptr(), lib.ptr(shift),
                     int(weight.dtype == torch.float32), lib.ptr(state if shift is not None else None), *seqs, S, slots, y.data_ptr(),
                     int(dt == torch.float32), T, D, groups, float(eps), lib.stream_ptr())
        lib.check_rc(rc, "lvb_depth_stream")
        return y
    x = history[0] if coef is None else torch.einsum("n,ntd->td", coef.float(), history)
    if out is not None:
        out.copy_(x)
    if rows is not None:
        x = x.index_select(0, rows.long())
    h = grouped_rms_norm(x, weight, eps, groups)
    if shift is None:
        return h.to(dt)
    y = h * (1.0 - shift.float())
    cu, lens, slot_ids = b.cu_q_lens.tolist(), b.seq_lens.tolist(), b.slot_ids.tolist()
    for i in range(int(b.num_seqs)):
        r0, r1 = cu[i], cu[i + 1]
        if r1 <= r0:
            continue
        known = 0 <= slot_ids[i] < state.shape[0]
        before = torch.zeros_like(h[r0:r1])
        before[1:] = h[r0:r1 - 1]
        if known and lens[i] > r1 - r0:
            before[0] = state[slot_ids[i]]
        y[r0:r1] = h[r0:r1] + (before - h[r0:r1]) * shift.float()
        if known:
            state[slot_ids[i]] = h[r1 - 1]
    return y.to(dt)
