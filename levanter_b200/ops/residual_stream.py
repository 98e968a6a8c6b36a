"""Pre-norm (and pre- and post-normed) blocks around an fp32 residual stream (``csrc/residual_stream.cu`` and the GEMM epilogues).

The stream ``x`` is an fp32 tensor whatever the model's compute dtype: the embedding starts it, RMS norms read it and hand the
compute dtype to the projections, and the projections that end a block accumulate into it in their epilogue.  Where a block's output is normed before it is added, the projection
hands it over in fp32 and :func:`add_norm_stream` norms it, adds it and norms the sum for the next block.  The kernels run
when no gradient is being recorded; with autograd the same steps are PyTorch ops on an fp32 stream, and on the CPU they are the
PyTorch statements only."""
from __future__ import annotations

from typing import Optional

import torch

from ..utils.activation import ActivationFunctionEnum
from . import lib
from .gemm import gemm, linear
from .glu import ClampedGlu, GatedActivation, gated_activation

_f = {}


def _kernels(*tensors) -> bool:
    """The in-place / fused kernels may run: CUDA tensors and nothing to differentiate."""
    return not torch.is_grad_enabled() and all(t.is_cuda for t in tensors) and lib.available()


def embed_stream(ids: torch.Tensor, weight: torch.Tensor, scale: float, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``scale * weight[ids]`` in fp32.  ``out``: where to (serving; contiguous fp32 rows)."""
    if _kernels(ids, weight) and weight.dtype in (torch.float32, torch.bfloat16) and weight.is_contiguous():
        c = lib
        if "e" not in _f:
            _f["e"] = lib.fn("lvb_embed_stream", [c.c_void_p, c.c_void_p, c.c_int, c.c_void_p, c.c_int, c.c_int, c.c_int, c.c_float,
                                                  c.c_void_p, c.c_void_p])
        flat = ids.reshape(-1).to(torch.int32).contiguous()
        V, D = weight.shape
        out = torch.empty(flat.numel(), D, dtype=torch.float32, device=weight.device) if out is None else out
        rc = _f["e"](flat.data_ptr(), weight.data_ptr(), int(weight.dtype == torch.float32), out.data_ptr(), flat.numel(), D, V, float(scale),
                     lib.status_buffer().data_ptr(), lib.stream_ptr())
        lib.check_rc(rc, "lvb_embed_stream")
        return out.view(*ids.shape, D)
    x = torch.nn.functional.embedding(ids.long(), weight).float() * scale
    return x if out is None else out.copy_(x.view_as(out)).view_as(x)


def rms_norm_stream(x: torch.Tensor, weight: torch.Tensor, eps: float, *, w_offset: float = 0.0, out_dtype: Optional[torch.dtype] = None,
                    rows: Optional[torch.Tensor] = None, add: Optional[torch.Tensor] = None) -> torch.Tensor:
    """RMS norm of the fp32 stream in ``out_dtype`` (default: the weight's dtype).  ``rows``: normalise these rows only.  ``add [D]``: a
    vector that joins every row of the stream first, in place (serving only)."""
    dt = out_dtype or weight.dtype
    if add is not None:
        assert rows is None and x.is_contiguous() and not torch.is_grad_enabled()
    if _kernels(x, weight) and (add is None or (add.is_contiguous() and add.dtype == weight.dtype)) and x.dtype == torch.float32 and dt in (torch.float32, torch.bfloat16) and weight.dtype in (torch.float32, torch.bfloat16) \
            and weight.is_contiguous():
        c = lib
        if "n" not in _f:
            _f["n"] = lib.fn("lvb_rms_stream", [c.c_void_p] * 4 + [c.c_int, c.c_void_p, c.c_int, c.c_int, c.c_int, c.c_float, c.c_float, c.c_void_p])
        D = x.shape[-1]
        x2 = x.reshape(-1, D)
        x2 = x2 if x2.is_contiguous() else x2.contiguous()
        if rows is not None:
            rows = rows.to(torch.int64).contiguous()
        n = x2.shape[0] if rows is None else rows.numel()
        y = torch.empty(n, D, dtype=dt, device=x.device)
        rc = _f["n"](x2.data_ptr(), lib.ptr(rows), lib.ptr(add), weight.data_ptr(), int(weight.dtype == torch.float32), y.data_ptr(), int(dt == torch.float32), n, D,
                     float(eps), float(w_offset), lib.stream_ptr())
        lib.check_rc(rc, "lvb_rms_stream")
        return y.view(*x.shape[:-1], D) if rows is None else y
    if add is not None:
        x.add_(add.float())
    if rows is not None:
        x = x.index_select(0, rows.long())
    xf = x.float()
    y = xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps) * (weight.float() + w_offset)
    return y.to(dt)


def add_norm_stream(x: torch.Tensor, y: torch.Tensor, w_post: torch.Tensor, w_next: torch.Tensor, eps: float, *,
                    rows: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Adds ``rms_norm(y) * w_post`` to the fp32 stream ``x`` in place and returns ``rms_norm(x) * w_next`` in the weights' dtype.
    ``rows``: the norm of these rows only; ``x`` is then left as it is (the last norm of a model)."""
    if _kernels(x, y, w_post, w_next) and x.dtype == y.dtype == torch.float32 and w_post.dtype == w_next.dtype and x.is_contiguous() \
            and w_post.dtype in (torch.float32, torch.bfloat16) and y.is_contiguous() and w_post.is_contiguous() and w_next.is_contiguous():
        c = lib
        if "an" not in _f:
            _f["an"] = lib.fn("lvb_add_norm_stream", [c.c_void_p] * 5 + [c.c_int, c.c_void_p] + [c.c_int] * 3 + [c.c_float, c.c_void_p])
        D = x.shape[-1]
        if rows is not None:
            rows = rows.to(torch.int64).contiguous()
        n = x.numel() // D if rows is None else rows.numel()
        h = torch.empty(n, D, dtype=w_next.dtype, device=x.device)
        f32 = int(w_next.dtype == torch.float32)
        rc = _f["an"](x.data_ptr(), y.data_ptr(), lib.ptr(rows), w_post.data_ptr(), w_next.data_ptr(), f32, h.data_ptr(), f32, n, D, float(eps),
                      lib.stream_ptr())
        lib.check_rc(rc, "lvb_add_norm_stream")
        return h.view(*x.shape[:-1], D) if rows is None else h
    if rows is not None:
        x, y = x.index_select(0, rows.long()), y.index_select(0, rows.long())
    x.add_(rms_norm_stream(y.float(), w_post, eps, out_dtype=torch.float32))
    return rms_norm_stream(x, w_next, eps)


_GLU_ANY = {ActivationFunctionEnum.gelu_new: 0, ActivationFunctionEnum.silu: 1, ActivationFunctionEnum.swish: 1}


def glu_of_rows(y: torch.Tensor, cols: int, act: GatedActivation, *, gate_logit: Optional[torch.Tensor] = None,
                out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    """``act(y[:, :cols]) * y[:, cols:2 * cols]`` of the joint product of a gate and an up projection, in ``out_dtype`` (default: ``y``'s).
    ``gate_logit [rows]``: every row is also multiplied by the sigmoid of its number."""
    gate, up = y[:, :cols], y[:, cols:2 * cols]
    dt = out_dtype or y.dtype
    plain = gate_logit is None and dt == y.dtype == torch.bfloat16 and cols % 8 == 0 and y.stride(0) % 8 == 0 and y.data_ptr() % 16 == 0
    clamped = isinstance(act, ClampedGlu)
    if (clamped or (act in _GLU_ANY and not plain)) and _kernels(y) \
            and y.dtype in (torch.float32, torch.bfloat16) and dt in (y.dtype, torch.bfloat16) and y.stride(1) == 1 \
            and (gate_logit is None or gate_logit.dtype == torch.float32):
        c = lib
        if "g" not in _f:
            _f["g"] = lib.fn("lvb_glu_any", [c.c_void_p] * 4 + [c.c_int, c.c_float] + [c.c_int] * 4 + [c.c_longlong] * 3 + [c.c_void_p])
        out = torch.empty(y.shape[0], cols, dtype=dt, device=y.device)
        rc = _f["g"](gate.data_ptr(), up.data_ptr(), lib.ptr(gate_logit), out.data_ptr(), 2 if clamped else _GLU_ANY[act],
                     act.limit if clamped else 0.0, int(y.dtype == torch.float32), int(dt == torch.float32), y.shape[0], cols, y.stride(0), y.stride(0), 0 if gate_logit is None else gate_logit.stride(0), lib.stream_ptr())
        lib.check_rc(rc, "lvb_glu_any")
        return out
    out = gated_activation(gate, up, act)
    if gate_logit is not None:
        out = out * torch.sigmoid(gate_logit.float())[:, None]
    return out.to(dt)


def _gemm_ok(h: torch.Tensor, w: torch.Tensor) -> bool:
    """The tcgen05 GEMM takes the product (forward only: the output size is free, the inner size a multiple of 8)."""
    return h.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and w.shape[1] % 8 == 0


def add_linear(x: torch.Tensor, h: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    """``x + h W^T`` on the fp32 stream.  Without autograd ``x`` itself is updated and returned."""
    if _kernels(x, h, weight):
        x2, h2 = x.view(-1, x.shape[-1]), h.reshape(-1, h.shape[-1])
        if _gemm_ok(h2, weight):
            gemm(h2, weight, out=x2, accumulate=True)
        elif h.dtype == torch.float32 and weight.dtype == torch.float32:
            x2.addmm_(h2, weight.t())
        else:
            x2.add_(torch.nn.functional.linear(h2, weight))
        return x
    return x + linear(h, weight).float()


def project(h: torch.Tensor, weight: torch.Tensor, *, bias: Optional[torch.Tensor] = None, squared_relu: bool = False,
            out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    """``h W^T + b`` (``max(., 0)^2`` of it), in ``h``'s dtype or in fp32 straight from the accumulator."""
    if _kernels(h, weight) and _gemm_ok(h, weight):
        h2 = h.reshape(-1, h.shape[-1])
        y = gemm(h2, weight, out_dtype=out_dtype or h.dtype, bias=bias, squared_relu=squared_relu)
        return y.view(*h.shape[:-1], weight.shape[0])
    if out_dtype == torch.float32 and h.dtype != torch.float32:
        # sizes the GEMM does not take (or with autograd, or on the CPU): the product itself in fp32
        y = torch.nn.functional.linear(h.float(), weight.float(), None if bias is None else bias.float())
    else:
        y = linear(h, weight, bias)
        if out_dtype is not None:
            y = y.to(out_dtype)
    return torch.relu(y).square() if squared_relu else y
