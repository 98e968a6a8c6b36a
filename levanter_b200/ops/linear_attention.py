"""Linear attention with a fixed decay per head (``csrc/linear_attention.cu``): ``S_t = decay S_{t-1} + k_t v_t^T``, ``o_t = S_t^T q_t`` with a matrix
state per head, and the norm and gate that follow it.

:func:`linear_attention_packed` is the serving form: packed rows of several sequences with a state per sequence slot.
:func:`fixed_decay_attention` is the differentiable form for whole sequences."""
from __future__ import annotations

import ctypes
from typing import Optional

import torch

from . import lib
from .depth_stream import grouped_rms_norm

CHUNK = 64
_f = {}


def fixed_decay_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor, segments: Optional[torch.Tensor] = None,
                          chunk: int = CHUNK) -> torch.Tensor:
    """``q, k [B, L, H, d]``, ``v [B, L, H, dv]``, ``decay [H]`` -> ``o [B, L, H, dv]`` in fp32.  ``segments [B, L]``: runs of equal ids are sequences
    of their own, each starting from a zero state.  By chunks: within one the products of all rows, between them the state."""
    B, L, H, d = q.shape
    q, k, v = (t.float().transpose(1, 2) for t in (q, k, v))
    S = q.new_zeros(B, H, d, v.shape[-1])
    i = torch.arange(chunk, device=q.device)
    g = decay.to(q.device, torch.float32)[:, None]
    outs = []
    for at in range(0, L, chunk):
        qc, kc, vc = (t[:, :, at:at + chunk] for t in (q, k, v))
        n = qc.shape[2]
        back = i[:n, None] - i[None, :n]
        D = torch.where(back >= 0, g[:, :, None] ** back.clamp_min(0), torch.zeros((), device=q.device))  # [H, n, n]
        reads, kept, stays = g ** (i[:n] + 1), g ** (n - 1 - i[:n]), g ** n  # [H, n], [H, n], [H, 1]
        D, reads, kept, stays = D[None], reads[None], kept[None], stays[None]
        if segments is not None:
            seg = segments[:, at:at + chunk]
            D = D * (seg[:, None, :, None] == seg[:, None, None, :])
            entered = segments[:, at - 1:at] if at else seg[:, :1]  # whose state comes in
            reads = reads * (seg == entered)[:, None]
            kept = kept * (seg == seg[:, -1:])[:, None]
            stays = stays * (seg[:, -1:] == entered)[:, None]
        outs.append((qc @ S) * reads[..., None] + ((qc @ kc.transpose(-1, -2)) * D) @ vc)
        S = S * stays[..., None] + (kc * kept[..., None]).transpose(-1, -2) @ vc
    return torch.cat(outs, dim=2).transpose(1, 2)


def _chunked_ok(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor) -> bool:
    d, dv = q.shape[2], v.shape[2]
    return q.dtype == torch.bfloat16 and d <= 256 and d % 8 == 0 and dv % 8 == 0 and q.stride(0) % 8 == 0 and all(t.data_ptr() % 16 == 0 for t in (q, k, v))


def linear_attention_packed(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor, state: torch.Tensor, batch_info, *,
                            key_scale: float = 1.0, silu: bool = False, chunked: Optional[bool] = None,
                            piece: Optional[int] = None) -> torch.Tensor:
    """``q, k [T, H, d]``, ``v [T, H, dv]`` (slices of the same packed rows) -> ``[T, H, dv]``; ``state [slots, H, d, dv]`` fp32, updated in place.
    ``key_scale``: factor on the keys.  ``silu``: q, k and v pass through it first (and may be overwritten).  A sequence whose first packed
    row is its position 0 starts from a zero state; rows of no sequence come out as zeros.  ``chunked``: by chunks on tensor cores (default:
    when sequences have many rows, in bf16, with sizes that are multiples of 8 and ``d`` up to 256), else row by row in fp32 arithmetic
    (``d`` up to 512).  ``piece``: rows (a multiple of 128) that the chunked form cuts longer sequences into, to walk the pieces at once
    (default: what should be fastest)."""
    T, H, d = q.shape
    dv = v.shape[2]
    b = batch_info
    if not torch.is_grad_enabled() and q.is_cuda and lib.available() and q.dtype in (torch.bfloat16, torch.float32) and state.is_contiguous() \
            and k.dtype == v.dtype == q.dtype and q.stride(0) == k.stride(0) == v.stride(0) \
            and all(t.stride(2) == 1 and t.stride(1) == t.shape[2] for t in (q, k, v)):
        c = lib
        if "l" not in _f:
            _f["l"] = lib.fn("lvb_linear_attention", [c.c_void_p] * 11 + [c.c_int] * 4 + [c.c_longlong] + [c.c_int] * 3 + [c.c_float] + [c.c_int] * 3 + [c.c_void_p] * 2)
            _f["plan"] = lib.fn("lvb_linear_attention_plan", [c.c_int] * 5 + [c.c_void_p] * 2, launches=0)
        i32 = lambda t: t.to(device=q.device, dtype=torch.int32).contiguous()  # noqa: E731
        slots, lens, cu, ns = i32(b.slot_ids), i32(b.seq_lens), i32(b.cu_q_lens), i32(b.num_seqs.reshape(1))
        S = slots.shape[0]
        longest = getattr(b, "longest", 0)
        if chunked is None:
            chunked = longest > 16 if longest > 0 else T > 4 * S
        chunked = chunked and _chunked_ok(q, k, v)
        cut, items = ctypes.c_int(piece or 0), ctypes.c_int(-(-T // piece) + min(S, T) if piece else 0)
        pieces = None
        if chunked:
            if piece is None:
                lib.check_rc(_f["plan"](T, longest, H, dv, S, ctypes.addressof(cut), ctypes.addressof(items)), "lvb_linear_attention_plan")
            if items.value:
                pieces = torch.empty(items.value * H * d * dv, dtype=torch.float32, device=q.device)
            if silu:
                silu_in_place(q, k, v)
        out = torch.empty(T, H, dv, dtype=q.dtype, device=q.device)
        rc = _f["l"](q.data_ptr(), k.data_ptr(), v.data_ptr(), out.data_ptr(), decay.data_ptr(), state.data_ptr(), slots.data_ptr(), lens.data_ptr(),
                     cu.data_ptr(), ns.data_ptr(), lib.ptr(pieces), T, H, d, dv, q.stride(0), S, state.shape[0], cut.value, float(key_scale),
                     int(silu and not chunked), int(q.dtype == torch.float32), int(chunked), lib.status_buffer().data_ptr(), lib.stream_ptr())
        lib.check_rc(rc, "lvb_linear_attention")
        return out
    act = torch.nn.functional.silu if silu else (lambda t: t)
    qf, kf, vf = act(q.float()), act(k.float()) * key_scale, act(v.float())
    g = decay.to(q.device, torch.float32)[:, None, None]
    out = torch.zeros(T, H, dv, dtype=torch.float32, device=q.device)
    cu, lens, slots = b.cu_q_lens.tolist(), b.seq_lens.tolist(), b.slot_ids.tolist()
    for i in range(int(b.num_seqs)):
        r0, r1 = cu[i], cu[i + 1]
        if r1 <= r0 or not 0 <= slots[i] < state.shape[0]:
            continue
        st = state[slots[i]].clone() if lens[i] > r1 - r0 else torch.zeros_like(state[slots[i]])
        for r in range(r0, r1):
            st = g * st + kf[r, :, :, None] * vf[r, :, None, :]
            out[r] = torch.einsum("hdv,hd->hv", st, qf[r])
        state[slots[i]] = st
    return out.to(q.dtype)


def silu_in_place(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor) -> None:
    """``silu`` of three slices of the same rows, in one pass where they lie side by side."""
    c = lib
    if "s" not in _f:
        _f["s"] = lib.fn("lvb_silu_rows", [c.c_void_p, c.c_longlong] + [c.c_int] * 3 + [c.c_void_p])
    size = q.element_size()
    spans = []
    for t in (q, k, v):
        at, n = t.data_ptr(), t.shape[1] * t.shape[2]
        if spans and spans[-1][0] + spans[-1][1] * size == at:
            spans[-1][1] += n
        else:
            spans.append([at, n])
    for at, n in spans:
        lib.check_rc(_f["s"](at, q.stride(0), q.shape[0], n, int(q.dtype == torch.float32), lib.stream_ptr()), "lvb_silu_rows")


def gated_norm(o: torch.Tensor, gate: torch.Tensor, eps: float, *, groups: int, weight: Optional[torch.Tensor] = None,
               sigmoid: bool = False) -> torch.Tensor:
    """``o [T, D]`` normed in groups (:func:`~.depth_stream.grouped_rms_norm`; ``weight`` None: ones), times ``silu(gate)`` (``sigmoid``: times its
    sigmoid), in ``o``'s dtype; ``gate [T, D]`` may be a slice of wider rows."""
    T, D = o.shape
    if not torch.is_grad_enabled() and o.is_cuda and lib.available() and o.dtype == gate.dtype and o.dtype in (torch.bfloat16, torch.float32) \
            and o.is_contiguous() and gate.stride(1) == 1 and (weight is None or weight.dtype in (torch.bfloat16, torch.float32)):
        c = lib
        if "g" not in _f:
            _f["g"] = lib.fn("lvb_gated_norm", [c.c_void_p] * 2 + [c.c_longlong, c.c_void_p, c.c_int, c.c_void_p] + [c.c_int] * 4 + [c.c_float, c.c_int, c.c_void_p])
        y = torch.empty_like(o)
        rc = _f["g"](o.data_ptr(), gate.data_ptr(), gate.stride(0), lib.ptr(weight), int(weight is not None and weight.dtype == torch.float32), y.data_ptr(),
                     int(o.dtype == torch.float32), T, D, groups, float(eps), int(sigmoid), lib.stream_ptr())
        lib.check_rc(rc, "lvb_gated_norm")
        return y
    n = grouped_rms_norm(o, torch.ones((), device=o.device) if weight is None else weight, eps, groups)
    g = torch.sigmoid(gate.float())
    return (n * (g if sigmoid else gate.float() * g)).to(o.dtype)
