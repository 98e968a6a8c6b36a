"""Flash attention on tcgen05 tensor cores (``csrc/flash_attn*.cu``): head sizes 64 and 128, causal (with sliding window) or
not, GQA, segment ids, any sequence length (padded to a multiple of 128 behind a segment id of its own).

Replaces the reference's fused-attention call sites (TransformerEngine/cuDNN on GPU, src/levanter/layers/attention.py:
533-544; pure-JAX flash attention, src/levanter/models/flash_attention.py:143-385)."""
from __future__ import annotations

import math
from typing import Optional

import torch

from . import lib
from .map_difference import MapDifference


def kernel_built() -> bool:
    try:
        return hasattr(lib.load(), "lvb_flash_attn_fwd")
    except Exception:
        return False


def supported(q, k, v, mask, bias, no_dropout: bool, attention_dtype) -> bool:
    from ..layers.attention import AttentionMask, _structured_only

    if not (q.is_cuda and lib.available() and kernel_built()):
        return False
    if bias is not None or not no_dropout:
        return False
    if q.dtype != torch.bfloat16 or k.dtype != torch.bfloat16 or v.dtype != torch.bfloat16:
        return False
    if attention_dtype is not None and attention_dtype not in (torch.float32, torch.bfloat16):
        return False
    if q.shape[-1] not in (64, 128) or v.shape[-1] != q.shape[-1] or k.shape[-1] != q.shape[-1]:
        return False
    if mask is not None and not isinstance(mask, AttentionMask):
        return False
    if q.shape[1] != k.shape[1] and (q.shape[1] == 1 or (isinstance(mask, AttentionMask) and mask.is_causal)):
        return False  # different query and key lengths: cross attention only (no causal part); single-token decode steps stay off
    if isinstance(mask, AttentionMask) and not mask.is_causal and mask.sliding_window:
        return False
    if isinstance(mask, AttentionMask) and mask.chunk_size is not None and q.shape[1] != k.shape[1]:
        return False
    return _structured_only(mask)


_packed = {}


def packed_supported(q, k, v, scale: float, maps: int = 1) -> bool:
    """Shapes :func:`flash_attention_packed` takes: bf16 rows on a B200, sizes that are multiples of 8 (keys up to 192, with two score maps up
    to 128; values up to 128), a positive scale (the running maximum is taken over unscaled scores) and 16-byte aligned rows."""
    most = 192 if maps == 1 else 128
    return packed_rows_ok(q, most) and packed_rows_ok(k, most) and packed_rows_ok(v, 128) and q.shape[0] % 256 == 0 and scale > 0.0


def packed_rows_ok(t: torch.Tensor, most: int) -> bool:
    """Rows ``t [T, heads, size]`` that the packed kernel's tensor maps can describe, with a size of at most ``most``."""
    return (t.is_cuda and lib.available() and t.dtype == torch.bfloat16 and t.shape[2] % 8 == 0 and t.shape[2] <= most and t.stride(2) == 1
            and t.stride(1) == t.shape[2] and t.stride(0) % 8 == 0 and t.data_ptr() % 16 == 0)


def flash_attention_packed(q, k, v, pos, *, scaling_factor: float, chunk: Optional[int] = None, window: Optional[int] = None, gate=None,
                           logits_soft_cap: Optional[float] = None, sink: Optional[torch.Tensor] = None,
                           difference: Optional[MapDifference] = None) -> torch.Tensor:
    """Causal attention over packed rows of sequences that start at position 0: ``q [T, Hq, dk]``, ``k [T, Hkv, dk]``, ``v [T, Hkv, dv]``
    (slices of one wider row are fine), ``pos [T]`` int32 positions with padding rows at 0, ``T`` a multiple of 256 ->
    ``[T, Hq, dv]``.  ``chunk``: a row sees its own chunk of that many positions only.  ``window``: a row sees itself and the
    ``window - 1`` positions before it.  ``gate [T, Hq * dv]`` or ``[T, Hq]``: the result is multiplied by its sigmoid.  ``sink [Hq]`` (fp32):
    a number per head that joins the softmax denominator as it is.  ``difference``: ``q [T, 2 Hq, dk]`` and ``k [T, 2 Hkv, dk]`` hold the two
    score maps of a head side by side, and their results are combined.  Forward only; shapes as in :func:`packed_supported`."""
    c = lib
    if "f" not in _packed:
        _packed["f"] = lib.fn("lvb_flash_attn_fwd_packed", [c.c_void_p] * 7 + [c.c_int] * 12 + [c.c_float, c.c_float, c.c_void_p, c.c_float, c.c_float,
                                                                                               c.c_void_p, c.c_void_p])
    T, rows, dk = q.shape
    Hq = rows if difference is None else rows // 2
    Hkv, dv = v.shape[1], v.shape[2]
    if difference is not None and sink is not None:
        raise NotImplementedError("differential attention takes no sink")
    pos = pos.to(torch.int32).contiguous()
    ldg = per_head = 0
    if gate is not None:
        per_head = int(gate.shape[1] == Hq)
        if gate.dtype != torch.bfloat16 or gate.stride(1) != 1 or (not per_head and (gate.stride(0) % 8 != 0 or gate.data_ptr() % 16 != 0)):
            gate = gate.to(torch.bfloat16).contiguous()
        ldg = gate.stride(0)
    diff = (0, 0.0, 0.0) if difference is None else (difference.weight.data_ptr(), float(difference.scale), float(difference.eps))
    out = torch.empty(T, Hq, dv, dtype=torch.bfloat16, device=q.device)
    rc = _packed["f"](q.data_ptr(), k.data_ptr(), v.data_ptr(), lib.ptr(gate), lib.ptr(sink), out.data_ptr(), pos.data_ptr(), T, Hq, Hkv, dk, dv, q.stride(0),
                      k.stride(0), v.stride(0), ldg, per_head, int(chunk or 0), int(window or 0), float(scaling_factor), float(logits_soft_cap or 0.0),
                      *diff, lib.status_buffer().data_ptr(), lib.stream_ptr())
    lib.check_rc(rc, "lvb_flash_attn_fwd_packed")
    return out


def flash_attention(q, k, v, mask, *, logits_soft_cap: Optional[float] = None, scaling_factor: Optional[float] = None, sink=None):
    from ._flash_impl import flash_attention_cuda

    return flash_attention_cuda(q, k, v, mask, logits_soft_cap=logits_soft_cap, scaling_factor=scaling_factor, sink=sink)
