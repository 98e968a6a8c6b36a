"""Paged-KV attention for the inference engine: KV page write and ragged paged attention
(src/levanter/layers/attention.py:1694-1695 and :1856-1991).

On a B200 both run as CUDA kernels (``csrc/paged_attention.cu``) that read sequence boundaries and lengths from device
arrays, so a decode step never synchronises with the host.  The PyTorch statements below are the CPU path and the test
oracle."""
from __future__ import annotations

import math
from typing import Optional

import torch

from . import lib
from .map_difference import MapDifference

INVALID = 2_000_000
_f = {}
_scratch = {}


def _use_kernel(*tensors) -> bool:
    return all(t.is_cuda for t in tensors) and lib.available()


def kv_page_write(kv_pages: torch.Tensor, new_k: torch.Tensor, new_v: torch.Tensor, dests: torch.Tensor) -> None:
    """Write ``new_k/new_v [T, KV, D]`` to flat slots ``dests[T]`` (= page * page_size + slot) of
    ``kv_pages[P, page_size, 2*KV, D]``; K goes to even head indices, V to odd.  Out-of-range slots are dropped."""
    P, ps, H2, D = kv_pages.shape
    if _use_kernel(kv_pages, new_k, new_v, dests) and kv_pages.dtype == torch.bfloat16 and D % 8 == 0:
        c = lib
        if "w" not in _f:
            _f["w"] = lib.fn("lvb_kv_page_write", [c.c_void_p] * 4 + [c.c_int] * 3 + [c.c_longlong, c.c_void_p])
        k = new_k.to(torch.bfloat16).contiguous()
        v = new_v.to(torch.bfloat16).contiguous()
        d = dests.to(torch.int32).contiguous()
        rc = _f["w"](kv_pages.data_ptr(), k.data_ptr(), v.data_ptr(), d.data_ptr(), k.shape[0], H2 // 2, D, P * ps, lib.stream_ptr())
        lib.check_rc(rc, "lvb_kv_page_write")
        return
    flat = kv_pages.view(P * ps, H2, D)
    valid = (dests >= 0) & (dests < P * ps)
    sel = valid.nonzero().squeeze(-1)
    idx = dests[sel].long()
    flat[idx, 0::2] = new_k[sel].to(kv_pages.dtype)
    flat[idx, 1::2] = new_v[sel].to(kv_pages.dtype)


def ragged_paged_attention(q: torch.Tensor, kv_pages: torch.Tensor, kv_lens: torch.Tensor, page_indices: torch.Tensor,
                           cu_q_lens: torch.Tensor, num_seqs, sm_scale: float = 1.0, soft_cap: Optional[float] = None) -> torch.Tensor:
    """Causal attention of packed query tokens ``q[T, H, D]`` over each sequence's pages.

    Sequence ``i`` owns query rows ``cu_q_lens[i]:cu_q_lens[i+1]``; its keys are the first ``kv_lens[i]`` slots of pages
    ``page_indices[i]``; query ``j`` of the sequence sits at absolute position ``kv_lens[i] - q_len + j``.  Rows past
    ``cu_q_lens[num_seqs]`` are padding and come back as zeros."""
    T, H, D = q.shape
    P, ps, H2, _ = kv_pages.shape
    KV = H2 // 2
    if _use_kernel(q, kv_pages) and q.dtype == torch.bfloat16 and kv_pages.dtype == torch.bfloat16 and D in (64, 128, 256) \
            and H // KV <= 16:
        return _paged_attention_cuda(q, kv_pages, kv_lens, page_indices, cu_q_lens, num_seqs, sm_scale, soft_cap)
    return ragged_paged_attention_reference(q, kv_pages, kv_lens, page_indices, cu_q_lens, num_seqs, sm_scale, soft_cap)


def _paged_attention_cuda(q, kv_pages, kv_lens, page_indices, cu_q_lens, num_seqs, sm_scale, soft_cap):
    c = lib
    if "a" not in _f:
        _f["a"] = lib.fn("lvb_paged_attention", [c.c_void_p] * 9 + [c.c_int] * 8 + [c.c_float, c.c_float, c.c_void_p], launches=2)
        _f["parts"] = lib.fn("lvb_paged_attention_parts", [c.c_int], launches=0)
    T, H, D = q.shape
    P, ps, H2, _ = kv_pages.shape
    S, PP = page_indices.shape
    dev = q.device
    i32 = lambda t: t.to(device=dev, dtype=torch.int32).contiguous()  # noqa: E731
    ns = num_seqs if isinstance(num_seqs, torch.Tensor) else torch.tensor(int(num_seqs), dtype=torch.int32)
    ns = i32(ns.reshape(1))
    parts = _f["parts"](PP * ps)
    key = (dev, T, H, parts, D)
    if parts > 1 and key not in _scratch:
        _scratch.clear()  # one live shape at a time: the engine calls with fixed T per phase
        _scratch[key] = (torch.empty(T * H * parts * D, dtype=torch.float32, device=dev),
                         torch.empty(T * H * parts * 2, dtype=torch.float32, device=dev))
    po, pml = _scratch.get(key, (None, None))
    qc = q.contiguous()
    out = torch.empty_like(qc)
    rc = _f["a"](qc.data_ptr(), kv_pages.data_ptr(), i32(kv_lens).data_ptr(), i32(page_indices).data_ptr(), i32(cu_q_lens).data_ptr(),
                 ns.data_ptr(), out.data_ptr(), lib.ptr(po), lib.ptr(pml), T, H, H2 // 2, D, S, PP, ps, P, float(sm_scale),
                 float(soft_cap or 0.0), lib.stream_ptr())
    lib.check_rc(rc, "lvb_paged_attention")
    return out


# ------------------------------------------------------------------------------------------------ general form
# Key and value sizes of their own, attention within chunks of positions or a sliding window, an output gate, fp32.  The cache of a layer is then viewed
# as [page, slot, kv_head, k_size + v_size], which for equal sizes is the memory of [page, slot, 2 * kv_head, size].
def _kv_view(kv_pages: torch.Tensor, kv_heads: int, k_size: int, v_size: int) -> torch.Tensor:
    return kv_pages.view(kv_pages.shape[0], kv_pages.shape[1], kv_heads, k_size + v_size)


def _strided_rows(t: torch.Tensor, n: int) -> torch.Tensor:
    """``t [T, heads, size]`` with heads and sizes packed inside a row (a row stride is fine)."""
    return t if t.stride(2) == 1 and t.stride(1) == t.shape[2] and (t.shape[0] <= 1 or t.stride(0) >= n) else t.contiguous()


def kv_page_write_general(kv_pages: torch.Tensor, new_k: torch.Tensor, new_v: torch.Tensor, dests: torch.Tensor) -> None:
    """:func:`kv_page_write` for ``new_k [T, KV, k_size]`` and ``new_v [T, KV, v_size]`` (rows may be strided) in bf16 or fp32."""
    KV, dk, dv = new_k.shape[1], new_k.shape[2], new_v.shape[2]
    kv = _kv_view(kv_pages, KV, dk, dv)
    slots = kv.shape[0] * kv.shape[1]
    if _use_kernel(kv_pages, new_k, new_v, dests):
        c = lib
        if "wg" not in _f:
            _f["wg"] = lib.fn("lvb_kv_page_write_general", [c.c_void_p] * 4 + [c.c_int] * 4 + [c.c_longlong] * 3 + [c.c_int, c.c_void_p])
        dt = kv.dtype
        k, v = _strided_rows(new_k.to(dt), KV * dk), _strided_rows(new_v.to(dt), KV * dv)
        d = dests.to(torch.int32).contiguous()
        rc = _f["wg"](kv.data_ptr(), k.data_ptr(), v.data_ptr(), d.data_ptr(), k.shape[0], KV, dk, dv, k.stride(0), v.stride(0), slots,
                      int(dt == torch.float32), lib.stream_ptr())
        lib.check_rc(rc, "lvb_kv_page_write_general")
        return
    sel = ((dests >= 0) & (dests < slots)).nonzero().squeeze(-1)
    flat = kv.view(slots, KV, dk + dv)
    flat[dests[sel].long()] = torch.cat([new_k[sel], new_v[sel]], dim=-1).to(kv.dtype)


def _gate_args(gate: Optional[torch.Tensor], dtype: torch.dtype, heads: int, v_size: int):
    """``(gate as the kernels take it, row stride, whether it has one number per head)`` of a gate ``[T, heads * v_size]`` or ``[T, heads]``."""
    if gate is None:
        return None, 0, 0
    assert gate.shape[1] in (heads, heads * v_size)
    gate = gate if gate.stride(1) == 1 and gate.dtype == dtype else gate.to(dtype).contiguous()
    return gate, gate.stride(0), int(gate.shape[1] == heads)


def _apply_gate(out: torch.Tensor, gate: torch.Tensor) -> torch.Tensor:
    """``out [T, heads, v_size]`` times the sigmoid of either form of gate."""
    return out * torch.sigmoid(gate.float()).view(out.shape[0], out.shape[1], -1)


def _difference_args(d: Optional[MapDifference]):
    return (0, 0.0, 0.0) if d is None else (d.weight.data_ptr(), float(d.scale), float(d.eps))


def paged_attention_general(q: torch.Tensor, kv_pages: torch.Tensor, kv_heads: int, v_size: int, batch_info, *, sm_scale: float,
                            chunk: Optional[int] = None, window: Optional[int] = None, gate: Optional[torch.Tensor] = None,
                            soft_cap: Optional[float] = None, difference: Optional[MapDifference] = None) -> torch.Tensor:
    """:func:`ragged_paged_attention` of ``q [T, H, k_size]`` (rows may be strided) over pages of ``kv_heads * (k_size + v_size)``
    elements per slot -> ``[T, H, v_size]``.

    ``chunk``: positions are cut into chunks of that many, counted from the start of the sequence, and a query sees the keys of
    its own chunk only.  ``window``: a query sees itself and the ``window - 1`` positions before it.  ``gate [T, H * v_size]`` or
    ``[T, H]``: the result is multiplied by its sigmoid.  ``difference``: rows ``2h`` and ``2h + 1`` of ``q`` are the two score maps of head
    ``h``, a slot holds ``2 * k_size + v_size`` elements per KV head, and the maps' results are combined -> ``[T, H / 2, v_size]``.  bf16
    with sizes that are multiples of 8 up to 256 (with two maps: the sum of both keys) and at most 16 query rows per KV head runs
    on tensor cores; everything else in fp32 arithmetic."""
    T, rows, dk = q.shape
    maps = 1 if difference is None else 2
    H = rows // maps
    b = batch_info
    if not _use_kernel(q, kv_pages):
        return paged_attention_general_reference(q, kv_pages, kv_heads, v_size, b, sm_scale=sm_scale, chunk=chunk, window=window, gate=gate,
                                                 soft_cap=soft_cap, difference=difference)
    kv = _kv_view(kv_pages, kv_heads, maps * dk, v_size)
    if kv.dtype not in (torch.bfloat16, torch.float32):
        raise TypeError(f"the cache must be bf16 or fp32, got {kv.dtype}")
    q = q.to(kv.dtype)  # attention runs in the cache's type
    c = lib
    P, ps = kv.shape[:2]
    S, PP = b.page_indices.shape
    dev = q.device
    i32 = lambda t: t.to(device=dev, dtype=torch.int32).contiguous()  # noqa: E731
    lens, pages, cu = i32(b.seq_lens), i32(b.page_indices), i32(b.cu_q_lens)
    ns = i32(b.num_seqs.reshape(1))
    q = _strided_rows(q, rows * dk)
    gate, ldg, per_head = _gate_args(gate, q.dtype, H, v_size)
    diff = _difference_args(difference)
    out = torch.empty(T, H, v_size, dtype=q.dtype, device=dev)
    tensor_cores = (q.dtype == torch.bfloat16 and dk % 8 == 0 and v_size % 8 == 0 and max(maps * dk, v_size) <= 256 and rows // kv_heads <= 16
                    and q.stride(0) % 2 == 0 and q.data_ptr() % 4 == 0)
    if not tensor_cores:
        scratch = None if difference is None else torch.empty(T * rows * v_size, dtype=torch.float32, device=dev)
        rc = _any_fn()(q.data_ptr(), kv.data_ptr(), lens.data_ptr(), pages.data_ptr(), cu.data_ptr(), ns.data_ptr(), lib.ptr(gate), 0, out.data_ptr(),
                       lib.ptr(scratch), T, rows, kv_heads, dk, v_size, q.stride(0), ldg, per_head, S, PP, ps, P, int(chunk or 0), int(window or 0), 0,
                       float(sm_scale), float(soft_cap or 0.0), *diff, int(q.dtype == torch.float32), lib.stream_ptr())
        lib.check_rc(rc, "lvb_attention_any")
        return out
    if "g" not in _f:
        _f["g"] = lib.fn("lvb_paged_attention_general", [c.c_void_p] * 10 + [c.c_int] * 14 + [c.c_float, c.c_float, c.c_void_p, c.c_float, c.c_float, c.c_void_p],
                         launches=2)
        _f["gparts"] = lib.fn("lvb_paged_attention_general_parts", [c.c_int] * 3, launches=0)
    parts = _f["gparts"](PP * ps, int(chunk or 0), int(window or 0))
    po = pml = None
    if parts > 1:
        po, pml = _part_scratch(dev, T * rows * parts * v_size, T * rows * parts * 2)
    rc = _f["g"](q.data_ptr(), kv.data_ptr(), lens.data_ptr(), pages.data_ptr(), cu.data_ptr(), ns.data_ptr(), lib.ptr(gate), out.data_ptr(), lib.ptr(po),
                 lib.ptr(pml), T, rows, kv_heads, dk, v_size, q.stride(0), ldg, per_head, S, PP, ps, P, int(chunk or 0), int(window or 0),
                 float(sm_scale), float(soft_cap or 0.0), *diff, lib.stream_ptr())
    lib.check_rc(rc, "lvb_paged_attention_general")
    return out


def _any_fn():
    if "any" not in _f:
        c = lib
        _f["any"] = lib.fn("lvb_attention_any", [c.c_void_p] * 10 + [c.c_int] * 5 + [c.c_longlong] * 2 + [c.c_int] * 8 +
                           [c.c_float, c.c_float, c.c_void_p, c.c_float, c.c_float, c.c_int, c.c_void_p])
    return _f["any"]


_part = {}


def _part_scratch(dev, n_o: int, n_ml: int):
    """Scratch for the partitions' partial results, grown as needed and shared by every layer: on one stream a layer's merge has
    consumed it before the next layer's partitions are written.  A buffer that grew stays referenced, because a captured graph
    may still write to the smaller one."""
    bufs = _part.setdefault(dev, [])
    for o, ml in bufs:
        if o.numel() >= n_o and ml.numel() >= n_ml:
            return o, ml
    pair = (torch.empty(n_o, dtype=torch.float32, device=dev), torch.empty(n_ml, dtype=torch.float32, device=dev))
    bufs.append(pair)
    return pair


def paged_attention_general_reference(q, kv_pages, kv_heads: int, v_size: int, batch_info, *, sm_scale: float, chunk: Optional[int] = None,
                                      window: Optional[int] = None, gate: Optional[torch.Tensor] = None, soft_cap: Optional[float] = None,
                                      shared: bool = False, difference: Optional[MapDifference] = None,
                                      sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """PyTorch statement of :func:`paged_attention_general` and, with ``shared``, of :func:`paged_attention_latent` (CPU path and test
    oracle).  ``shared``: a KV head's row is its key, whose first ``v_size`` elements are the value."""
    T, H, dk = q.shape
    maps = 1 if difference is None else 2
    b = batch_info
    kv_all = _kv_view(kv_pages, kv_heads, maps * dk, 0 if shared else v_size)
    v_at = 0 if shared else maps * dk
    ps = kv_all.shape[1]
    G = H // kv_heads  # query rows per KV head: its query heads, with two maps (head, map)
    out = torch.zeros(T, H, v_size, dtype=torch.float32, device=q.device)
    cu, lens = b.cu_q_lens.tolist(), b.seq_lens.tolist()
    for i in range(int(b.num_seqs)):
        q0, q1, kl = cu[i], cu[i + 1], lens[i]
        if q1 <= q0 or kl <= 0 or kl == INVALID:
            continue
        n = (kl + ps - 1) // ps
        kv = kv_all[b.page_indices[i, :n].long()].reshape(n * ps, kv_heads, -1)[:kl].float()
        keys = kv[..., :maps * dk].unflatten(2, (maps, dk))
        qi = q[q0:q1].float().view(q1 - q0, kv_heads, G // maps, maps, dk)
        s = (torch.einsum("qkgmd,skmd->kgmqs", qi, keys) * sm_scale).flatten(1, 2)
        if soft_cap:
            s = torch.tanh(s / soft_cap) * soft_cap
        qpos = torch.arange(q1 - q0, device=q.device) + (kl - (q1 - q0))
        kpos = torch.arange(kl, device=q.device)
        see = kpos[None, :] <= qpos[:, None]
        if chunk:
            see = see & (kpos[None, :] // chunk == qpos[:, None] // chunk)
        if window:
            see = see & (qpos[:, None] - kpos[None, :] < window)
        s = s.masked_fill(~see, -float("inf"))
        if sink is not None:  # one more column, without a value
            s = torch.cat([s, sink.float().view(kv_heads, G, 1, 1).expand(kv_heads, G, q1 - q0, 1)], dim=-1)
        p = torch.softmax(s, dim=-1)[..., :kl]
        out[q0:q1] = torch.einsum("kgqs,skd->qkgd", p, kv[..., v_at:v_at + v_size]).reshape(q1 - q0, H, v_size)
    if difference is not None:
        out = difference(out[:, 0::2], out[:, 1::2])
    if gate is not None:
        out = _apply_gate(out, gate)
    return out.to(q.dtype)


# ------------------------------------------------------------------------------------------------ latent form
def paged_attention_latent(q: torch.Tensor, kv_pages: torch.Tensor, rank: int, batch_info, *, sm_scale: float,
                           window: Optional[int] = None, sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal attention of ``q [T, H, width]`` over pages of ``width`` elements per slot whose first ``rank`` are the value: all heads read
    the same row per key -> ``[T, H, rank]``.  ``window`` as in :func:`paged_attention_general`.  ``sink [H]`` (fp32): one number per head
    that joins the softmax denominator as it is, without a key or a value.  bf16 with sizes that are multiples of
    8 (rank up to 512, width up to 576) runs on tensor cores; everything else in fp32 arithmetic."""
    T, H, w = q.shape
    b = batch_info
    if not _use_kernel(q, kv_pages):
        return paged_attention_general_reference(q, kv_pages, 1, rank, b, sm_scale=sm_scale, window=window, shared=True, sink=sink)
    kv = kv_pages.view(kv_pages.shape[0], kv_pages.shape[1], w)
    if kv.dtype not in (torch.bfloat16, torch.float32):
        raise TypeError(f"the cache must be bf16 or fp32, got {kv.dtype}")
    q = q.to(kv.dtype).contiguous()
    c = lib
    P, ps = kv.shape[:2]
    S, PP = b.page_indices.shape
    dev = q.device
    i32 = lambda t: t.to(device=dev, dtype=torch.int32).contiguous()  # noqa: E731
    lens, pages, cu, ns = i32(b.seq_lens), i32(b.page_indices), i32(b.cu_q_lens), i32(b.num_seqs.reshape(1))
    out = torch.empty(T, H, rank, dtype=q.dtype, device=dev)
    if q.dtype != torch.bfloat16 or w % 8 != 0 or rank % 8 != 0 or rank > 512 or w > 576:
        rc = _any_fn()(q.data_ptr(), kv.data_ptr(), lens.data_ptr(), pages.data_ptr(), cu.data_ptr(), ns.data_ptr(), 0, lib.ptr(sink), out.data_ptr(), 0, T, H,
                       1, w, rank, H * w, 0, 0, S, PP, ps, P, 0, int(window or 0), 1, float(sm_scale), 0.0, 0, 0.0, 0.0, int(q.dtype == torch.float32),
                       lib.stream_ptr())
        lib.check_rc(rc, "lvb_attention_any")
        return out
    if "l" not in _f:
        _f["l"] = lib.fn("lvb_paged_latent", [c.c_void_p] * 10 + [c.c_int] * 10 + [c.c_float, c.c_void_p, c.c_void_p], launches=2)
        _f["lparts"] = lib.fn("lvb_paged_latent_parts", [c.c_int] * 6, launches=0)
    parts = _f["lparts"](T, H, w, rank, PP * ps, int(window or 0))
    po = pml = None
    if parts > 1:
        po, pml = _part_scratch(dev, T * H * parts * rank, T * H * parts * 2)
    rc = _f["l"](q.data_ptr(), kv.data_ptr(), lens.data_ptr(), pages.data_ptr(), cu.data_ptr(), ns.data_ptr(), lib.ptr(sink), out.data_ptr(), lib.ptr(po), lib.ptr(pml), T,
                 H, w, rank, S, PP, ps, P, int(window or 0), parts, float(sm_scale), lib.status_buffer().data_ptr(), lib.stream_ptr())
    lib.check_rc(rc, "lvb_paged_latent")
    return out


def head_product(a: torch.Tensor, b: torch.Tensor, out: torch.Tensor, *, b_trans: bool, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``out[t, h] = a[t, h] b[h]`` (``b [H, K, N]``) or ``a[t, h] b[h]^T`` (``b_trans``, ``b [H, N, K]``) for ``a [T, H, K]``, written into
    ``out [T, H, N]``; all three may be strided views with packed last dimensions.  ``gate [T, H * N]``: the result is multiplied by its
    sigmoid."""
    T, H, K = a.shape
    N = out.shape[2]
    kernel = (_use_kernel(a, b, out) and a.dtype == b.dtype == out.dtype == torch.bfloat16 and a.stride(2) == b.stride(2) == out.stride(2) == 1
              and not any(v % 8 for v in (N, K, a.stride(0), a.stride(1), b.stride(0), b.stride(1), out.stride(0), out.stride(1)))
              and a.data_ptr() % 16 == 0 and b.data_ptr() % 16 == 0
              and (gate is None or (gate.dtype == a.dtype and gate.stride(1) == 1 and gate.stride(0) % 2 == 0 and gate.data_ptr() % 4 == 0)))
    if not kernel:
        y = torch.matmul(a.transpose(0, 1), b.transpose(1, 2) if b_trans else b).transpose(0, 1)
        out.copy_(y if gate is None else _apply_gate(y.float(), gate))
        return out
    c = lib
    if "hp" not in _f:
        _f["hp"] = lib.fn("lvb_head_product", [c.c_void_p] * 4 + [c.c_int] * 4 + [c.c_longlong] * 7 + [c.c_int, c.c_void_p])
    rc = _f["hp"](a.data_ptr(), b.data_ptr(), out.data_ptr(), lib.ptr(gate), T, H, N, K, a.stride(0), a.stride(1), b.stride(1), b.stride(0), out.stride(0),
                  out.stride(1), 0 if gate is None else gate.stride(0), int(b_trans), lib.stream_ptr())
    lib.check_rc(rc, "lvb_head_product")
    return out


def ragged_paged_attention_reference(q, kv_pages, kv_lens, page_indices, cu_q_lens, num_seqs, sm_scale: float = 1.0,
                                     soft_cap: Optional[float] = None) -> torch.Tensor:
    T, H, D = q.shape
    P, ps, H2, _ = kv_pages.shape
    KV = H2 // 2
    G = H // KV
    out = torch.zeros_like(q)
    n = int(num_seqs)
    cu = cu_q_lens.tolist()
    lens = kv_lens.tolist()
    for i in range(n):
        q0, q1 = cu[i], cu[i + 1]
        ql = q1 - q0
        kl = lens[i]
        if ql <= 0 or kl <= 0 or kl == INVALID:
            continue
        npages = (kl + ps - 1) // ps
        pages = page_indices[i, :npages].long()
        kv = kv_pages[pages].reshape(npages * ps, H2, D)[:kl]
        k = kv[:, 0::2].float()
        v = kv[:, 1::2].float()
        qi = q[q0:q1].float().view(ql, KV, G, D) * sm_scale
        s = torch.einsum("qkgd,skd->kgqs", qi, k)
        if soft_cap is not None and soft_cap > 0:
            s = torch.tanh(s / soft_cap) * soft_cap
        qpos = torch.arange(ql, device=q.device) + (kl - ql)
        kpos = torch.arange(kl, device=q.device)
        s = s.masked_fill(~(qpos[:, None] >= kpos[None, :]), -float("inf"))
        p = torch.softmax(s, dim=-1)
        o = torch.einsum("kgqs,skd->qkgd", p, v)
        out[q0:q1] = o.reshape(ql, H, D).to(q.dtype)
    return out
