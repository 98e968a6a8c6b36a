"""Between the projections of an attention layer and attention itself, over the packed rows of a serving step: rotary positions, score
temperatures, value mixing, the norm of a compressed row, and the write into the paged cache, in one kernel (``csrc/qkv_prep.cu``).

The kernels run when no gradient is being recorded; the PyTorch statements are the CPU path and the test oracle."""
from __future__ import annotations

from typing import Optional, Tuple

import torch

from ..layers.rotary import RotaryEmbeddings
from . import lib
from .paged_attention import _strided_rows, kv_page_write_general

_f = {}


def _kernel(*tensors) -> bool:
    return not torch.is_grad_enabled() and all(t.is_cuda for t in tensors) and lib.available() and tensors[0].dtype in (torch.bfloat16, torch.float32)


def _i32(t: torch.Tensor) -> torch.Tensor:
    return t.to(torch.int32).contiguous()


def _rotation_args(rot: Optional[RotaryEmbeddings], device):
    if rot is None:
        return 0, 0, 0, 1.0, 1.0
    return rot.frequencies_on(device).data_ptr(), rot.rotary_dim, int(rot.interleaved), float(rot.position_scale), float(rot.temperature)


def mix_values(v: torch.Tensor, v_first: torch.Tensor, mix: torch.Tensor) -> torch.Tensor:
    """``(1 - mix) v + mix v_first`` in fp32, in ``v``'s dtype."""
    m = mix.float()
    return ((1.0 - m) * v.float() + m * v_first.float()).to(v.dtype)


def prepare_qkv(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, kv_pages: torch.Tensor, dests: torch.Tensor, pos: torch.Tensor, *,
                rot: Optional[RotaryEmbeddings] = None, head_scale: Optional[torch.Tensor] = None, v_first: Optional[torch.Tensor] = None,
                mix: Optional[torch.Tensor] = None) -> Tuple[torch.Tensor, torch.Tensor, torch.Tensor]:
    """``q [T, H, dk]``, ``k [T, KV * n, dk]``, ``v [T, KV, dv]`` (strided rows; they may be updated in place) -> what attention reads:
    ``q`` and ``k`` rotated by ``rot`` at ``pos``, ``q`` times ``head_scale[h]``, ``v`` mixed with ``v_first [T, KV, dv]``.  ``k`` and ``v``
    are also written to slots ``dests`` of the cache: per KV head its ``n`` keys (one per score map), then its value."""
    T, H, dk = q.shape
    KV, dv = v.shape[1], v.shape[2]
    maps = k.shape[1] // KV
    dt = q.dtype
    small = [t for t in (head_scale, mix) if t is not None]
    if _kernel(q, k, v, kv_pages) and k.dtype == v.dtype == kv_pages.dtype == dt and all(t.dtype in (torch.bfloat16, torch.float32) for t in small) \
            and len({t.dtype for t in small}) <= 1 and (v_first is None or v_first.dtype == dt):
        q, k, v = _strided_rows(q, H * dk), _strided_rows(k, KV * maps * dk), _strided_rows(v, KV * dv)
        if v_first is not None:
            v_first = _strided_rows(v_first, KV * dv)
        c = lib
        if "q" not in _f:
            _f["q"] = lib.fn("lvb_qkv_prep", [c.c_void_p] * 9 + [c.c_int] * 6 + [c.c_longlong] * 5 + [c.c_void_p, c.c_int, c.c_int, c.c_float, c.c_float,
                                                                                                    c.c_int, c.c_int, c.c_void_p])
        d, p = _i32(dests), _i32(pos)
        hs = None if head_scale is None else head_scale.contiguous()
        slots = kv_pages.shape[0] * kv_pages.shape[1]
        rc = _f["q"](q.data_ptr(), k.data_ptr(), v.data_ptr(), lib.ptr(v_first), lib.ptr(mix if v_first is not None else None), lib.ptr(hs),
                     kv_pages.data_ptr(), p.data_ptr(), d.data_ptr(), T, H, KV, maps, dk, dv, q.stride(0), k.stride(0), v.stride(0),
                     0 if v_first is None else v_first.stride(0), slots, *_rotation_args(rot, q.device), int(dt == torch.float32),
                     int(bool(small) and small[0].dtype == torch.float32), lib.stream_ptr())
        lib.check_rc(rc, "lvb_qkv_prep")
        return q, k, v
    qf = q.float() if rot is None else rot(q.float(), pos)
    if head_scale is not None:
        qf = qf * head_scale.float()[:, None]
    if rot is not None:
        k = rot(k, pos)
    if v_first is not None:
        v = mix_values(v, v_first, mix)
    kv_page_write_general(kv_pages, k.reshape(T, KV, maps * dk), v, dests)
    return qf.to(dt), k, v


def _latent_fn():
    if "l" not in _f:
        c = lib
        _f["l"] = lib.fn("lvb_latent_prep", [c.c_void_p] * 8 + [c.c_int] * 4 + [c.c_longlong] * 6 + [c.c_float, c.c_void_p, c.c_int, c.c_float, c.c_float,
                                                                                                   c.c_int, c.c_int, c.c_void_p])
    return _f["l"]


def prepare_latent(down: torch.Tensor, norm_weight: torch.Tensor, eps: float, kv_pages: torch.Tensor, dests: torch.Tensor, pos: torch.Tensor,
                   rot: Optional[RotaryEmbeddings], q_rot: torch.Tensor, q_out: Optional[torch.Tensor] = None,
                   to_cache_only: bool = False) -> Tuple[Optional[torch.Tensor], torch.Tensor]:
    """``down [T, rank + r]``: a compressed row and a key part of ``r`` dimensions shared by the heads (0, and no ``rot``: there is none).  Returns ``(latent, q_out)``:
    ``latent [T, rank + r]`` is the RMS norm of the former (weight ``norm_weight [rank]``) and the latter rotated at ``pos``, also written
    to slots ``dests`` of the cache; the heads' query parts ``q_rot [T, H, r]`` are rotated into ``q_out`` (None: in place).
    ``to_cache_only``: the caller does not read ``latent``, which may come back as None."""
    T, width = down.shape
    rank, r = norm_weight.shape[0], width - norm_weight.shape[0]
    dt = down.dtype
    dst = q_rot if q_out is None else q_out
    assert (rot.rotary_dim if rot is not None else 0) == r, "the shared key part is rotated as a whole"
    if _kernel(down, norm_weight, kv_pages, q_rot, dst) and q_rot.dtype == dst.dtype == kv_pages.dtype == dt and down.stride(1) == 1 \
            and norm_weight.dtype in (torch.bfloat16, torch.float32) and q_rot.stride(2) == dst.stride(2) == 1:
        latent = None if to_cache_only and rot is None else torch.empty(T, width, dtype=dt, device=down.device)
        d, p, w = _i32(dests), _i32(pos), norm_weight.contiguous()
        freq, dims, inter, pscale, mag = _rotation_args(rot, down.device)
        rc = _latent_fn()(down.data_ptr(), w.data_ptr(), lib.ptr(latent), kv_pages.data_ptr(), q_rot.data_ptr(), dst.data_ptr(), p.data_ptr(), d.data_ptr(), T,
                     q_rot.shape[1], rank, r, down.stride(0), q_rot.stride(0), q_rot.stride(1), dst.stride(0), dst.stride(1),
                     kv_pages.shape[0] * kv_pages.shape[1], float(eps), freq, inter, pscale, mag, int(dt == torch.float32), int(w.dtype == torch.float32),
                     lib.stream_ptr())
        lib.check_rc(rc, "lvb_latent_prep")
        return latent, dst
    x = down[:, :rank].float()
    c = (x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * norm_weight.float()).to(dt)
    latent = c if rot is None else torch.cat([c, rot(down[:, None, rank:], pos)[:, 0]], dim=1)
    flat = kv_pages.view(-1, width)
    sel = ((dests >= 0) & (dests < flat.shape[0])).nonzero().squeeze(-1)
    flat[dests[sel].long()] = latent[sel].to(flat.dtype)
    if rot is not None:
        dst.copy_(rot(q_rot, pos))
    return latent, dst


def rotate_queries(q_rot: torch.Tensor, pos: torch.Tensor, rot: RotaryEmbeddings, q_out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """The query half of :func:`prepare_latent`, for layers that read rows which another layer has cached: ``q_rot [T, H, r]`` rotated at ``pos``
    into ``q_out`` (None: in place)."""
    T, H, r = q_rot.shape
    dst = q_rot if q_out is None else q_out
    assert rot.rotary_dim == r
    if _kernel(q_rot, dst) and q_rot.dtype == dst.dtype and q_rot.stride(2) == dst.stride(2) == 1:
        p = _i32(pos)
        freq, _, inter, pscale, mag = _rotation_args(rot, q_rot.device)
        rc = _latent_fn()(0, 0, 0, 0, q_rot.data_ptr(), dst.data_ptr(), p.data_ptr(), 0, T, H, 0, r, 0, q_rot.stride(0), q_rot.stride(1), dst.stride(0),
                          dst.stride(1), 0, 0.0, freq, inter, pscale, mag, int(q_rot.dtype == torch.float32), 0, lib.stream_ptr())
        lib.check_rc(rc, "lvb_latent_prep")
        return dst
    dst.copy_(rot(q_rot, pos))
    return dst


def norm_rows(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """RMS norm of ``x [T, width]``, a slice of wider rows (a compressed row on its way to the next projection) -> ``[T, width]`` packed."""
    T, width = x.shape
    if _kernel(x, weight) and x.stride(1) == 1 and weight.dtype in (torch.bfloat16, torch.float32):
        y, w = torch.empty(T, width, dtype=x.dtype, device=x.device), weight.contiguous()
        rc = _latent_fn()(x.data_ptr(), w.data_ptr(), y.data_ptr(), 0, 0, 0, 0, 0, T, 1, width, 0, x.stride(0), 0, 0, 0, 0, 0, float(eps), 0, 0, 1.0, 1.0,
                          int(x.dtype == torch.float32), int(w.dtype == torch.float32), lib.stream_ptr())
        lib.check_rc(rc, "lvb_latent_prep")
        return y
    f = x.float()
    return (f * torch.rsqrt(f.pow(2).mean(-1, keepdim=True) + eps) * weight.float()).to(x.dtype)
