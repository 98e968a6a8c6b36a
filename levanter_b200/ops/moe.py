"""Grouped (per-expert) SwiGLU MLP over rows sorted by expert: the reference's three ``hnn.MoELinear`` ragged dots
(src/levanter/models/mixtral.py:245-277).

Rows ``[sum(group_sizes), hidden]`` are contiguous per expert.  Each expert's slice runs through the tcgen05 GEMM
(gate and up projections, the gated-activation kernel, then the down projection); expert boundaries are read back once
per call."""
from __future__ import annotations

import torch

from ..utils.activation import ActivationFunctionEnum
from .gemm import linear
from .glu import GatedActivation, gated_activation


def grouped_mlp(x_sorted: torch.Tensor, group_sizes: torch.Tensor, w1: torch.Tensor, w3: torch.Tensor, w2: torch.Tensor,
                act: ActivationFunctionEnum, first_expert: int = 0) -> torch.Tensor:
    """``out[rows of expert e] = (act(x w1[e]^T) * (x w3[e]^T)) w2[e]^T``; ``w1/w3: [E, mlp, hidden]``, ``w2: [E, hidden, mlp]``.
    ``group_sizes`` covers the experts held in ``w*`` starting at global expert ``first_expert``."""
    sizes = group_sizes.tolist()
    n_local = w1.shape[0]
    sizes = sizes[first_expert:first_expert + n_local] if len(sizes) != n_local else sizes
    outs = []
    start = 0
    dt = x_sorted.dtype
    for e, n in enumerate(sizes):
        if n == 0:
            continue
        xe = x_sorted[start:start + n]
        a, b, c = w1[e], w3[e], w2[e]
        if a.dtype != dt:
            a, b, c = a.to(dt), b.to(dt), c.to(dt)
        h = gated_activation(linear(xe, a), linear(xe, b), act)
        outs.append(linear(h, c))
        start += n
    if not outs:
        return x_sorted.new_zeros((0, w2.shape[1]))
    return torch.cat(outs, dim=0)


# ------------------------------------------------------------------------------------------------ padded grouped path
# Rows sorted by expert with every expert's segment padded to a multiple of 128 rows: no row block of the GEMM kernel
# straddles two experts, the expert boundaries stay on the device (no host read-back, so the step can be captured in a
# CUDA graph), and one launch covers all experts (``lvb_gemm_grouped``).
BLOCK = 128


def padded_layout(expert_of_row: torch.Tensor, num_experts: int):
    """For ``expert_of_row[R]`` (the expert each (token, choice) pair goes to) returns, all on the device:
    ``dest[R]``: row of every pair in the padded sorted buffer; ``offsets[E + 1]``: padded start row of every expert;
    ``tile_group[capacity / 128]``: expert of every 128-row block (-1 past the end); and the static ``capacity``."""
    R = expert_of_row.numel()
    E = num_experts
    capacity = ((R + E * (BLOCK - 1)) + BLOCK - 1) // BLOCK * BLOCK
    idx = expert_of_row.reshape(-1).long()
    counts = torch.bincount(idx, minlength=E)
    padded = (counts + BLOCK - 1) // BLOCK * BLOCK
    offsets = torch.zeros(E + 1, dtype=torch.long, device=idx.device)
    offsets[1:] = torch.cumsum(padded, 0)
    starts = torch.zeros(E, dtype=torch.long, device=idx.device)
    starts[1:] = torch.cumsum(counts, 0)[:-1]
    order = torch.argsort(idx, stable=True)
    rank_sorted = torch.empty_like(order)
    rank_sorted[order] = torch.arange(R, device=idx.device)
    dest = offsets[idx] + (rank_sorted - starts[idx])
    blocks = torch.arange(capacity // BLOCK, device=idx.device)
    tile_group = torch.searchsorted(offsets[1:] // BLOCK, blocks, right=True)
    tile_group = torch.where(blocks < offsets[E] // BLOCK, tile_group, torch.full_like(tile_group, -1))
    return dest, offsets.to(torch.int32), tile_group.to(torch.int32), capacity


def _grouped_fn():
    from . import lib

    c = lib
    return lib.fn("lvb_gemm_grouped", [c.c_int, c.c_void_p, c.c_void_p, c.c_void_p] + [c.c_int] * 9 + [c.c_float, c.c_void_p, c.c_void_p,
                                                                                                     c.c_void_p, c.c_void_p])


_g = {}


def _grouped(kind, a, b, out, groups, Tp, M, N, K, flags, tile_group, offsets):
    from . import lib

    if "f" not in _g:
        _g["f"] = _grouped_fn()
    rc = _g["f"](kind, a.data_ptr(), b.data_ptr(), out.data_ptr(), groups, Tp, M, N, K, a.stride(0), b.stride(-2), out.stride(-2), flags, 1.0,
                 lib.ptr(tile_group), lib.ptr(offsets), lib.status_buffer().data_ptr(), lib.stream_ptr())
    lib.check_rc(rc, "lvb_gemm_grouped")
    return out


def _use_grouped_kernel(x: torch.Tensor, w: torch.Tensor) -> bool:
    from . import lib

    return x.is_cuda and lib.available() and x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and w.shape[1] % BLOCK == 0 \
        and w.shape[2] % 8 == 0


class _GroupedLinear(torch.autograd.Function):
    """``y[rows of expert e] = x[rows of e] w[e]^T`` over the padded layout; ``w``: ``[E, out, in]``."""

    @staticmethod
    def forward(ctx, x, w, tile_group, offsets):
        E, N, K = w.shape
        Tp = x.shape[0]
        y = torch.empty(Tp, N, dtype=x.dtype, device=x.device)
        _grouped(0, x, w, y, E, Tp, 0, N, K, 0, tile_group, None)
        ctx.save_for_backward(x, w, tile_group, offsets)
        return y

    @staticmethod
    def backward(ctx, dy):
        x, w, tile_group, offsets = ctx.saved_tensors
        E, N, K = w.shape
        Tp = x.shape[0]
        dy = dy.contiguous()
        dx = dw = None
        if ctx.needs_input_grad[0]:
            dx = torch.empty(Tp, K, dtype=x.dtype, device=x.device)
            _grouped(1, dy, w, dx, E, Tp, 0, K, N, 0, tile_group, None)
            # row blocks past the last expert were skipped by the kernel: their gradient is zero, not whatever the buffer held
            dx = torch.where((tile_group >= 0).repeat_interleave(BLOCK).unsqueeze(1), dx, torch.zeros((), dtype=dx.dtype, device=dx.device))
        if ctx.needs_input_grad[1]:
            main = getattr(w, "main_grad", None)
            if main is not None:
                _grouped(2, dy, x, main, E, Tp, N, K, 0, 1 | 2, None, offsets)  # fp32, accumulate into the engine's buffer
                dw = None
            else:
                acc = torch.zeros(E, N, K, dtype=torch.float32, device=x.device)
                _grouped(2, dy, x, acc, E, Tp, N, K, 0, 1 | 2, None, offsets)
                dw = acc.to(w.dtype)
        return dx, dw, None, None


def grouped_linear(x_pad: torch.Tensor, w: torch.Tensor, tile_group: torch.Tensor, offsets: torch.Tensor) -> torch.Tensor:
    if _use_grouped_kernel(x_pad, w):
        return _GroupedLinear.apply(x_pad, w, tile_group, offsets)
    # reference: one matmul per expert over its padded segment (CPU path and test oracle)
    off = offsets.tolist()
    y = x_pad.new_zeros(x_pad.shape[0], w.shape[1])
    for e in range(w.shape[0]):
        if off[e + 1] > off[e]:
            y[off[e]:off[e + 1]] = x_pad[off[e]:off[e + 1]] @ w[e].to(x_pad.dtype).t()
    return y


def grouped_mlp_padded(x_flat: torch.Tensor, topk_idx: torch.Tensor, w1: torch.Tensor, w3: torch.Tensor, w2: torch.Tensor,
                       act: ActivationFunctionEnum) -> torch.Tensor:
    """Expert MLP of every (token, choice) pair: ``x_flat[T, hidden]``, ``topk_idx[T, k]`` -> ``[T * k, hidden]`` in pair order.
    Permutation into the padded layout, three grouped GEMMs with the gated activation in between, permutation back."""
    T, k = topk_idx.shape
    E = w1.shape[0]
    dest, offsets, tile_group, capacity = padded_layout(topk_idx.reshape(-1), E)
    x_pad = x_flat.new_zeros(capacity, x_flat.shape[1])
    x_pad = x_pad.index_copy(0, dest, x_flat.repeat_interleave(k, dim=0))
    dt = x_flat.dtype
    if w1.dtype != dt:
        w1, w3, w2 = w1.to(dt), w3.to(dt), w2.to(dt)
    h = gated_activation(grouped_linear(x_pad, w1, tile_group, offsets), grouped_linear(x_pad, w3, tile_group, offsets), act)
    y = grouped_linear(h, w2, tile_group, offsets)
    return y.index_select(0, dest)


def grouped_mlp_on_padded(x_pad: torch.Tensor, tile_group: torch.Tensor, offsets: torch.Tensor, w1: torch.Tensor, w3: torch.Tensor,
                          w2: torch.Tensor, act: ActivationFunctionEnum) -> torch.Tensor:
    """The expert MLP over rows that are already in the padded expert-sorted layout (``offsets[E + 1]`` padded starts,
    ``tile_group`` the expert of every 128-row block, both on the device): what the expert-parallel exchange delivers."""
    dt = x_pad.dtype
    if w1.dtype != dt:
        w1, w3, w2 = w1.to(dt), w3.to(dt), w2.to(dt)
    h = gated_activation(grouped_linear(x_pad, w1, tile_group, offsets), grouped_linear(x_pad, w3, tile_group, offsets), act)
    return grouped_linear(h, w2, tile_group, offsets)


# ------------------------------------------------------------------------------------------------ routing
def moe_route_reference(router_logits: torch.Tensor, k: int):
    """``(topk_w[T, k], topk_idx[T, k], counts[E], p_sum[E], lse[T])`` with PyTorch ops (CPU path and oracle)."""
    z = router_logits.float()
    probs = torch.softmax(z, dim=-1)
    w, idx = torch.topk(probs, k, dim=-1)
    w = w / w.sum(-1, keepdim=True)
    counts = torch.bincount(idx.reshape(-1), minlength=z.shape[-1])
    return w, idx, counts, probs.sum(0), torch.logsumexp(z, dim=-1)


class _MoeRoute(torch.autograd.Function):
    @staticmethod
    def forward(ctx, logits, k):
        from . import lib

        c = lib
        T, E = logits.shape
        z = logits.float().contiguous()
        dev = z.device
        idx = torch.empty(T, k, dtype=torch.int32, device=dev)
        w = torch.empty(T, k, dtype=torch.float32, device=dev)
        probs = torch.empty(T, E, dtype=torch.float32, device=dev)
        lse = torch.empty(T, dtype=torch.float32, device=dev)
        counts = torch.zeros(E, dtype=torch.int32, device=dev)
        psum = torch.empty(E, dtype=torch.float32, device=dev)
        scratch = torch.empty(((T + 127) // 128) * E, dtype=torch.float32, device=dev)
        f = lib.fn("lvb_moe_route_fwd", [c.c_void_p, c.c_int, c.c_int, c.c_int] + [c.c_void_p] * 8, launches=2)
        rc = f(z.data_ptr(), T, E, k, idx.data_ptr(), w.data_ptr(), probs.data_ptr(), lse.data_ptr(), counts.data_ptr(), psum.data_ptr(),
               scratch.data_ptr(), lib.stream_ptr())
        lib.check_rc(rc, "lvb_moe_route_fwd")
        ctx.save_for_backward(probs, idx)
        ctx.k = k
        ctx.in_dtype = logits.dtype
        idx64 = idx.long()
        ctx.mark_non_differentiable(idx64, counts)
        return w, idx64, counts, psum, lse

    @staticmethod
    def backward(ctx, d_w, _d_idx, _d_counts, d_psum, d_lse):
        from . import lib

        c = lib
        probs, idx = ctx.saved_tensors
        T, E = probs.shape
        dz = torch.empty_like(probs)
        prep = lambda t: None if t is None else t.float().contiguous()  # noqa: E731
        d_w, d_psum, d_lse = prep(d_w), prep(d_psum), prep(d_lse)
        f = lib.fn("lvb_moe_route_bwd", [c.c_void_p] * 5 + [c.c_int] * 3 + [c.c_void_p, c.c_void_p])
        rc = f(probs.data_ptr(), idx.data_ptr(), lib.ptr(d_w), lib.ptr(d_psum), lib.ptr(d_lse), T, E, ctx.k, dz.data_ptr(), lib.stream_ptr())
        lib.check_rc(rc, "lvb_moe_route_bwd")
        return dz.to(ctx.in_dtype), None


def moe_route(router_logits: torch.Tensor, k: int):
    """Routing of ``router_logits[T, E]``: renormalised top-``k`` weights and indices, tokens per expert, per-expert sums of
    the router probabilities (for the load-balancing loss) and the per-token log-sum-exp (for the router z-loss).
    Differentiable in the weights, the probability sums and the log-sum-exp."""
    from . import lib

    E = router_logits.shape[-1]
    if router_logits.is_cuda and lib.available() and E <= 64 and k <= 8:
        return _MoeRoute.apply(router_logits, k)
    return moe_route_reference(router_logits, k)


# ------------------------------------------------------------------------------------------------ routing within groups, for serving
# The router scores experts by a sigmoid or a softmax, chooses by score (+ correction) within the best groups of neighbouring experts;
# experts are plain (squared ReLU) or gated (SiLU) layers.  ``csrc/moe_experts.cu``.
def _within_groups(choice: torch.Tensor, groups: int, keep: int, best: int) -> torch.Tensor:
    """``choice [T, E]`` with -inf outside the ``keep`` groups of neighbours whose ``best`` largest choice scores sum highest."""
    if groups <= 1 or keep >= groups:
        return choice
    T, E = choice.shape
    size = E // groups
    gs = choice.view(T, groups, size).topk(min(best, size), dim=-1).values.sum(-1)
    kept = torch.zeros(T, groups, dtype=torch.bool, device=choice.device)
    kept.scatter_(1, gs.topk(keep, dim=-1).indices, True)
    return choice.masked_fill(~kept.repeat_interleave(size, dim=1), float("-inf"))


def route_sigmoid_reference(logits: torch.Tensor, correction, k: int, groups: int, keep: int, scale: float):
    """``(idx[T, k], w[T, k])``: see :func:`route_sigmoid`.  Differentiable in the weights."""
    s = torch.sigmoid(logits.float())
    c = s.detach() if correction is None else s.detach() + correction.float()
    idx = _within_groups(c, groups, keep, 2).topk(k, dim=-1).indices
    return idx, s.gather(1, idx) * scale


def route_softmax_reference(logits: torch.Tensor, k: int, groups: int, keep: int, bias=None):
    """``(idx[T, k], w[T, k])``: see :func:`route_softmax`.  Differentiable in the weights."""
    s = torch.softmax(logits.float() if bias is None else logits.float() + bias.float(), dim=-1)
    idx = _within_groups(s.detach(), groups, keep, 1).topk(k, dim=-1).indices
    w = s.gather(1, idx)
    return idx, w / (w.sum(-1, keepdim=True) + 1e-20)


class RoutedTokens:
    """What routing leaves on the device for the expert products: choices, weights and tokens per expert."""

    def __init__(self, idx, w, counts):
        self.idx, self.w, self.counts = idx, w, counts


def _route(kind: int, logits, correction, k, groups, keep, scale, live, live_limit) -> RoutedTokens:
    from . import lib

    T, E = logits.shape
    if not (logits.is_cuda and lib.available()):
        idx, w = route_softmax_reference(logits, k, groups, keep, correction) if kind else route_sigmoid_reference(logits, correction, k, groups, keep, scale)
        idx = idx.to(torch.int32)
        if live is not None:
            dead = (live < 0) | (live >= live_limit)
            idx, w = idx.masked_fill(dead[:, None], -1), w.masked_fill(dead[:, None], 0.0)
        return RoutedTokens(idx, w, None)
    c = lib
    if "rs" not in _g:
        _g["rs"] = lib.fn("lvb_moe_route_grouped", [c.c_int, c.c_void_p, c.c_longlong, c.c_void_p, c.c_int, c.c_void_p] + [c.c_int] * 6 +
                          [c.c_float, c.c_void_p, c.c_void_p, c.c_void_p, c.c_void_p])
    dev = logits.device
    z = logits if logits.stride(1) == 1 else logits.contiguous()
    if correction is not None and correction.dtype not in (torch.float32, torch.bfloat16):
        correction = correction.float()
    idx = torch.empty(T, k, dtype=torch.int32, device=dev)
    w = torch.empty(T, k, dtype=torch.float32, device=dev)
    counts = torch.empty(2 * E, dtype=torch.int32, device=dev)
    rc = _g["rs"](kind, z.data_ptr(), z.stride(0), lib.ptr(correction), int(correction is not None and correction.dtype == torch.float32), lib.ptr(live),
                  int(live_limit), T, E, k, groups, keep, float(scale), idx.data_ptr(), w.data_ptr(), counts.data_ptr(), lib.stream_ptr())
    lib.check_rc(rc, "lvb_moe_route_grouped")
    return RoutedTokens(idx, w, counts)


def route_sigmoid(logits: torch.Tensor, correction, k: int, *, groups: int = 1, keep: int = 1, scale: float = 1.0, live=None,
                  live_limit: int = 0) -> RoutedTokens:
    """Routing of fp32 ``logits [T, E]``: the ``k`` experts with the largest ``sigmoid(logits) + correction`` among those of the
    ``keep`` (of ``groups``) neighbour groups whose two best choice scores sum highest; weights ``scale * sigmoid(logits)``.
    ``live [T]`` int32: tokens whose value lies outside ``[0, live_limit)`` are padding and are sent to no expert (index -1)."""
    return _route(0, logits, correction, k, groups, keep, scale, live, live_limit)


def route_softmax(logits: torch.Tensor, k: int, *, groups: int = 1, keep: int = 1, bias=None, live=None, live_limit: int = 0) -> RoutedTokens:
    """Routing of fp32 ``logits [T, E]`` (rows may be strided; plus ``bias [E]``): the ``k`` experts with the largest softmax scores among those
    of the ``keep`` (of ``groups``) neighbour groups whose best score is largest; weights are the chosen scores divided by their sum, which is
    the softmax over the chosen logits.  ``live`` as in :func:`route_sigmoid`."""
    return _route(1, logits, bias, k, groups, keep, 1.0, live, live_limit)


def _block_rows(pairs: int, experts: int) -> int:
    """Rows an expert's segment is padded to: the tensor core's 128 when experts get that many tokens, fewer in decode rounds,
    where the expert products are streams over the weights and padding rows only cost launch width."""
    mean = pairs / experts
    for rows in (16, 32, 64):
        if mean <= rows // 2:
            return rows
    return BLOCK


def grouped_product(a: torch.Tensor, w: torch.Tensor, tile_group: torch.Tensor, rows: int, sq_relu: bool) -> torch.Tensor:
    """``a[rows of block b] w[tile_group[b]]^T`` (``max(., 0)^2`` of it) over blocks of ``rows`` rows, forward only; ``w [E, out, in]``.
    bf16 with sizes that are multiples of 8 on tensor cores, otherwise fp32 arithmetic on blocks of 64."""
    from . import lib

    c = lib
    if "fma" not in _g:
        _g["fma"] = lib.fn("lvb_grouped_fma", [c.c_void_p] * 4 + [c.c_int] * 5 + [c.c_void_p])
        _g["sk"] = lib.fn("lvb_gemm_skinny_grouped", [c.c_void_p] * 3 + [c.c_int] * 9 + [c.c_float, c.c_void_p, c.c_void_p, c.c_void_p])
    E, n, k = w.shape
    w = w if w.is_contiguous() else w.contiguous()
    y = torch.empty(a.shape[0], n, dtype=a.dtype, device=a.device)
    if a.dtype != torch.bfloat16 or n % 8 or k % 8:
        assert rows == 64
        rc = _g["fma"](a.data_ptr(), w.data_ptr(), y.data_ptr(), tile_group.data_ptr(), a.shape[0], n, k, int(sq_relu),
                       int(a.dtype == torch.float32), lib.stream_ptr())
    elif rows == BLOCK:
        return _grouped(0, a, w, y, E, a.shape[0], 0, n, k, 32 if sq_relu else 0, tile_group, None)
    else:
        rc = _g["sk"](a.data_ptr(), w.data_ptr(), y.data_ptr(), E, a.shape[0], rows, n, k, k, k, n, 32 if sq_relu else 0, 1.0,
                      tile_group.data_ptr(), lib.status_buffer().data_ptr(), lib.stream_ptr())
    lib.check_rc(rc, "grouped expert product")
    return y


def add_expert_outputs(stream: torch.Tensor, h: torch.Tensor, routed: RoutedTokens, up: torch.Tensor, down: torch.Tensor, *,
                       gated: bool = False, act: GatedActivation = ActivationFunctionEnum.silu) -> torch.Tensor:
    """``stream[t] += sum_j w[t, j] * down[e] relu(up[e] h[t])^2`` with ``e = idx[t, j]``, in place on the fp32 stream; ``up [E, ff, width]``,
    ``down [E, width, ff]``.  ``gated``: ``up [E, 2 ff, width]`` holds a gate and an up projection, and the inner layer is ``act(gate h) *
    (up h)``.  Forward only, CUDA only: dispatch into the block-padded expert-sorted layout, two grouped products (the
    activation in the epilogue of the first, or a gated activation between them), combine."""
    from . import lib
    from .residual_stream import glu_of_rows

    c = lib
    T, k = routed.idx.shape
    E, width, ff = down.shape
    dev = h.device
    tma = h.dtype == torch.bfloat16 and up.dtype == torch.bfloat16 and width % 8 == 0 and ff % 8 == 0
    rows = _block_rows(T * k, E) if tma else 64  # 64: the tile of the fp32 product
    blocks = (T * k + min(E, T * k) * (rows - 1) + rows - 1) // rows
    if "d" not in _g:
        _g["d"] = lib.fn("lvb_moe_dispatch", [c.c_void_p, c.c_void_p] + [c.c_int] * 5 + [c.c_void_p, c.c_void_p, c.c_int] + [c.c_void_p] * 3)
        _g["c"] = lib.fn("lvb_moe_combine", [c.c_void_p, c.c_int, c.c_void_p, c.c_void_p] + [c.c_int] * 3 + [c.c_void_p, c.c_void_p])
    x_pad = torch.empty(blocks * rows, width, dtype=h.dtype, device=dev)
    dest = torch.empty(T, k, dtype=torch.int32, device=dev)
    tile_group = torch.empty(blocks, dtype=torch.int32, device=dev)
    h = h.contiguous()
    rc = _g["d"](routed.idx.data_ptr(), routed.counts.data_ptr(), T, k, E, rows, blocks, h.data_ptr(), x_pad.data_ptr(), width * h.element_size(),
                 dest.data_ptr(), tile_group.data_ptr(), lib.stream_ptr())
    lib.check_rc(rc, "lvb_moe_dispatch")

    a = grouped_product(x_pad, up.to(h.dtype), tile_group, rows, not gated)
    if gated:
        a = glu_of_rows(a, ff, act)
    y = grouped_product(a, down.to(h.dtype), tile_group, rows, False)
    rc = _g["c"](y.data_ptr(), int(y.dtype == torch.float32), dest.data_ptr(), routed.w.data_ptr(), T, k, width, stream.data_ptr(), lib.stream_ptr())
    lib.check_rc(rc, "lvb_moe_combine")
    return stream


def expert_outputs(h: torch.Tensor, idx: torch.Tensor, w: torch.Tensor, up: torch.Tensor, down: torch.Tensor, *, gated: bool = False,
                   act: GatedActivation = ActivationFunctionEnum.silu) -> torch.Tensor:
    """The sum :func:`add_expert_outputs` adds, as differentiable framework ops (training, and the CPU path): ``[T, width]`` fp32."""
    T, k = idx.shape
    keep = idx >= 0
    dest, offsets, tile_group, capacity = padded_layout(idx.clamp_min(0).reshape(-1), up.shape[0])
    x_pad = h.new_zeros(capacity, h.shape[1]).index_copy(0, dest, h.repeat_interleave(k, dim=0))
    a = grouped_linear(x_pad, up.to(h.dtype), tile_group, offsets)
    if gated:
        a = gated_activation(a[:, :down.shape[2]], a[:, down.shape[2]:], act)
    else:
        a = torch.relu(a).square()
    y = grouped_linear(a, down.to(h.dtype), tile_group, offsets).index_select(0, dest).view(T, k, -1)
    return (y.float() * (w.float() * keep).unsqueeze(-1)).sum(1)
