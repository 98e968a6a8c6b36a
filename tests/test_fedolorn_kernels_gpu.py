"""The kernels Fedolorn serves with, one mechanism at a time, against the plain statement in ``fedolorn_oracle``."""
import dataclasses

import numpy as np
import pytest
import torch

import fedolorn_oracle as O
from levanter_b200.ops import lib

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32


def _rel(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return float((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt().clamp_min(1e-9))


def _randn(*shape, seed=0, dtype=BF, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("dim", [336, 72, 50, 4096])
def test_embedding_and_norm_of_the_stream(dtype, dim):
    from levanter_b200.ops.residual_stream import embed_stream, rms_norm_stream

    table, w = _randn(61, dim, dtype=dtype), _randn(dim, seed=1, dtype=dtype, scale=0.3)
    ids = torch.tensor([0, 60, 7, 7, 33])
    with torch.no_grad():
        x = embed_stream(ids.cuda(), table.cuda(), 3.25)
        rows = torch.tensor([4, 1, 1], device="cuda")
        y = rms_norm_stream(x, w.cuda(), 0.02, w_offset=1.0)
        z = rms_norm_stream(x, w.cuda(), 0.02, w_offset=1.0, rows=rows)
    lib.check_status()
    want = O.scaled_embedding(table.double(), ids, 3.25)
    assert x.dtype == F32 and y.dtype == dtype
    assert _rel(x, want) < 1e-7
    n = O.offset_rms_norm(want, w.double(), 0.02)
    assert _rel(y, n) < (2e-7 if dtype == F32 else 3e-3) and _rel(z, n[rows.cpu()]) < (2e-7 if dtype == F32 else 3e-3)


@pytest.mark.parametrize("M", [1, 64, 130, 300, 1024])
@pytest.mark.parametrize("N,K", [(264, 328), (136, 64), (40, 1536), (512, 4096)])
def test_products_with_activation_and_accumulation(M, N, K):
    from levanter_b200.ops.residual_stream import add_linear, project

    h, w, x = _randn(M, K), _randn(N, K, seed=1, scale=K ** -0.5), _randn(M, N, seed=2, dtype=F32)
    with torch.no_grad():
        a = project(h.cuda(), w.cuda(), squared_relu=True)
        z = project(h.cuda(), w.cuda(), out_dtype=F32)
        s = add_linear(x.cuda(), h.cuda(), w.cuda())
    lib.check_status()
    p = h.double() @ w.double().T
    assert _rel(a, O.squared_relu(p)) < 4e-3
    assert z.dtype == F32 and _rel(z, p) < 2e-6
    assert s.dtype == F32 and _rel(s, x.double() + p) < 2e-6


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("E,groups,keep,top,scale", [(18, 3, 1, 5, 1.9), (12, 3, 2, 3, 1.0), (64, 8, 3, 8, 0.7), (6, 6, 2, 2, 1.3), (160, 1, 1, 6, 1.0),
                                                     (10, 5, 5, 1, 2.0), (256, 8, 4, 8, 1.2)])
def test_routing(dtype, E, groups, keep, top, scale):
    from levanter_b200.ops.moe import route_sigmoid

    T = 37
    z, corr = _randn(T, E, seed=E, dtype=F32), _randn(E, seed=E + 1, dtype=dtype, scale=0.6) - 0.4  # some choice scores are negative
    live = torch.arange(T, dtype=torch.int32)
    live[5], live[6] = -1, 2_000_000
    r = route_sigmoid(z.cuda(), corr.cuda(), top, groups=groups, keep=keep, scale=scale, live=live.cuda(), live_limit=1000)
    idx, w = O.route(z.double(), corr.double(), top, groups, keep, scale)
    ok = torch.ones(T, dtype=torch.bool)
    ok[5] = ok[6] = False
    assert torch.equal(r.idx.cpu()[ok].long(), idx[ok]) and _rel(r.w.cpu()[ok], w[ok]) < 1e-6
    assert bool((r.idx.cpu()[~ok] == -1).all()) and bool((r.w.cpu()[~ok] == 0).all())
    assert torch.equal(r.counts[:E].cpu().long(), torch.bincount(idx[ok].reshape(-1), minlength=E))


@pytest.mark.parametrize("dtype,width,ff,E", [(BF, 352, 72, 14), (BF, 72, 136, 6), (BF, 50, 30, 5), (F32, 96, 40, 7), (BF, 512, 384, 3)])
@pytest.mark.parametrize("T,k", [(1, 2), (9, 3), (150, 2), (700, 3)])
def test_expert_outputs(dtype, width, ff, E, T, k):
    from levanter_b200.ops.moe import RoutedTokens, add_expert_outputs, expert_outputs, route_sigmoid

    h, up = _randn(T, width, dtype=dtype), _randn(E, ff, width, seed=1, dtype=dtype, scale=width ** -0.5)
    down, x = _randn(E, width, ff, seed=2, dtype=dtype, scale=ff ** -0.5), _randn(T, width, seed=3, dtype=F32)
    z = _randn(T, E, seed=4, dtype=F32)
    z[: T // 2, 1] += 6.0  # a crowded expert
    with torch.no_grad():
        r = route_sigmoid(z.cuda(), None, k, scale=1.5)
        got = add_expert_outputs(x.cuda(), h.cuda(), r, up.cuda(), down.cuda())
    lib.check_status()
    idx, w = O.route(z.double(), torch.zeros(E, dtype=torch.float64), k, 1, 1, 1.5)
    want = torch.zeros(T, width, dtype=torch.float64)
    for e in range(E):
        y = O.feed_forward(h.double(), up[e].double(), down[e].double())
        for j in range(k):
            m = idx[:, j] == e
            want[m] += w[m, j][:, None] * y[m]
    assert _rel(got.cpu().double() - x.double(), want) < (1e-6 if dtype == F32 else 8e-3)
    assert isinstance(r, RoutedTokens)
    diff = expert_outputs(h.cuda(), r.idx, r.w, up.cuda(), down.cuda())  # the differentiable form agrees
    assert _rel(diff, want) < (1e-6 if dtype == F32 else 1e-2)


# ------------------------------------------------------------------------------------------------ attention
@dataclasses.dataclass
class _Batch:
    page_indices: torch.Tensor
    seq_lens: torch.Tensor
    cu_q_lens: torch.Tensor
    num_seqs: torch.Tensor
    new_token_dests: torch.Tensor


def _sequences(lens, H, G, dk, dv, dtype, seed=0):
    return [(_randn(n, H, dk, seed=seed + 3 * i, dtype=dtype), _randn(n, G, dk, seed=seed + 3 * i + 1, dtype=dtype),
             _randn(n, G, dv, seed=seed + 3 * i + 2, dtype=dtype)) for i, n in enumerate(lens)]


def _needles(seqs, chunk):
    """Around every chunk border, one key that scores far above all others for the queries near it: a mask that is one position
    off gives those rows another value altogether."""
    for q, k, v in seqs:
        n, H, dk = q.shape
        for b in range(chunk, n, chunk):
            for key in (b - 1, b):
                d = key % dk
                k[key] = 0.0
                k[key, :, d] = 12.0 if key == b else 10.0
                q[max(0, b - 1):b + 2, :, d] += 6.0
    return seqs


def _paged(seqs, ps, dtype, seed=0):
    """The sequences' keys and values in shuffled pages, and the batch description of their last ``q`` rows."""
    from levanter_b200.ops import paged_attention as PA

    G, dk, dv = seqs[0][1].shape[1], seqs[0][1].shape[2], seqs[0][2].shape[2]
    need = [-(-k.shape[0] // ps) for _, k, _ in seqs]
    P = sum(need) + 3
    perm = torch.randperm(P, generator=torch.Generator().manual_seed(seed)).tolist()
    kv = torch.full((P, ps, G, dk + dv), float("nan"), dtype=dtype, device="cuda")
    pages = torch.full((len(seqs) + 1, max(need) + 1), 2_000_000, dtype=torch.int32)
    for i, (_, k, v) in enumerate(seqs):
        mine = [perm.pop() for _ in range(need[i])]
        pages[i, :need[i]] = torch.tensor(mine)
        dest = torch.tensor([mine[j // ps] * ps + j % ps for j in range(k.shape[0])], dtype=torch.int32)
        dest = torch.cat([dest, torch.tensor([2_000_000, -1], dtype=torch.int32)]).cuda()  # two padding tokens
        wide = torch.zeros(k.shape[0] + 2, G * (dk + dv) + 8, dtype=dtype)
        wide[:-2, :G * dk], wide[:-2, G * dk:G * (dk + dv)] = k.flatten(1), v.flatten(1)
        wide = wide.cuda()
        PA.kv_page_write_general(kv, wide[:, :G * dk].unflatten(1, (G, dk)), wide[:, G * dk:G * (dk + dv)].unflatten(1, (G, dv)), dest)
    return kv, pages.cuda()


def _check_rows(got, want, dtype):
    got, want = got.double().cpu(), want.double()
    err = (got - want).abs().amax(dim=(1, 2))
    tol = (2e-5 if dtype == F32 else 3e-2) * float(want.abs().max())
    assert float(err.max()) < tol, (int(err.argmax()), float(err.max()), tol)


PAGED = [(BF, 6, 3, 96, 88, 180), (BF, 6, 2, 64, 64, 48), (BF, 8, 1, 128, 128, 300), (BF, 4, 4, 40, 72, 7), (BF, 8, 2, 128, 64, 520),
         (BF, 3, 1, 256, 192, 64), (BF, 4, 1, 192, 128, 90), (BF, 4, 2, 200, 88, 40),
         (BF, 2, 2, 20, 12, 33), (BF, 20, 1, 64, 64, 50), (F32, 6, 2, 104, 80, 170), (F32, 6, 3, 33, 17, 10),
         (BF, 4, 2, 64, 64, 5000), (BF, 16, 1, 24, 128, 257)]


@pytest.mark.parametrize("dtype,H,G,dk,dv,chunk", PAGED)
def test_paged_attention_in_chunks(dtype, H, G, dk, dv, chunk):
    """Decode rows at and around chunk and page borders, portions of several tokens, gate, strided rows."""
    from levanter_b200.ops import paged_attention as PA

    ps = 16
    lens = [1, 2, 2 * chunk, 2 * chunk + 1, chunk, 601, 32, 33] if chunk < 400 else [1, chunk + 1 if chunk < 600 else 700, 601, 32, 600]
    seqs = _needles(_sequences(lens, H, G, dk, dv, dtype, seed=dk), chunk)
    kv, pages = _paged(seqs, ps, dtype)
    qn = [1, 2, 1, 1, min(5, chunk), 40, 1, 3][:len(lens)]
    T = sum(qn) + 2
    q = torch.zeros(T, H * dk + 16, dtype=dtype)
    gate = _randn(T, H * dv + 8, seed=9, dtype=dtype)
    want = torch.zeros(T, H, dv, dtype=torch.float64)
    at = 0
    for (qs, k, v), n in zip(seqs, qn):
        q[at:at + n, :H * dk] = qs[-n:].flatten(1)
        full = O.grouped_query_attention(qs.double(), k.double(), v.double(), 0.35, chunk)[-n:]
        want[at:at + n] = O.output_gate(full, gate[at:at + n, :H * dv].double().view(n, H, dv))
        at += n
    cu = torch.tensor(np.concatenate([[0], np.cumsum(qn), [at + 2]]), dtype=torch.int32, device="cuda")
    sl = torch.tensor(lens + [2_000_000], dtype=torch.int32, device="cuda")
    b = _Batch(pages, sl, cu, torch.tensor(len(lens), dtype=torch.int32, device="cuda"), None)
    got = PA.paged_attention_general(q.cuda()[:, :H * dk].unflatten(1, (H, dk)), kv, G, dv, b, sm_scale=0.35, chunk=chunk, gate=gate.cuda()[:, :H * dv])
    torch.cuda.synchronize()
    assert bool((got[at:] == 0).all())  # padding rows
    _check_rows(got[:at], want[:at], dtype)


@pytest.mark.parametrize("H,G,dk,dv,chunk", [(6, 3, 96, 88, 180), (2, 1, 64, 64, 128), (2, 2, 128, 128, 5000), (4, 1, 40, 72, 7), (2, 2, 128, 64, 256),
                                             (3, 3, 8, 16, 50), (4, 2, 112, 120, 129), (2, 1, 64, 128, 100)])
def test_packed_prefill_in_chunks(H, G, dk, dv, chunk):
    from levanter_b200.ops import flash_attention as FA

    lens = [1, 130, 700, 2, 257]
    seqs = _needles(_sequences(lens, H, G, dk, dv, BF, seed=dv), chunk)
    n = sum(lens)
    T = -(-n // 256) * 256
    wide = torch.zeros(T, H * dk + G * dk + G * dv + H * dv, dtype=BF)
    pos = torch.zeros(T, dtype=torch.int32)
    gate = _randn(n, H * dv, seed=11)
    at, want = 0, []
    for q, k, v in seqs:
        m = q.shape[0]
        wide[at:at + m] = torch.cat([q.flatten(1), k.flatten(1), v.flatten(1), gate[at:at + m]], dim=1)
        pos[at:at + m] = torch.arange(m)
        a = O.grouped_query_attention(q.double(), k.double(), v.double(), 0.35, chunk)
        want.append(O.output_gate(a, gate[at:at + m].double().view(m, H, dv)))
        at += m
    w = wide.cuda()
    c = [0, H * dk, (H + G) * dk, (H + G) * dk + G * dv]
    q, k, v = w[:, :c[1]].unflatten(1, (H, dk)), w[:, c[1]:c[2]].unflatten(1, (G, dk)), w[:, c[2]:c[3]].unflatten(1, (G, dv))
    assert FA.packed_supported(q, k, v, 0.35)
    got = FA.flash_attention_packed(q, k, v, pos.cuda(), scaling_factor=0.35, chunk=chunk, gate=w[:, c[3]:])
    torch.cuda.synchronize()
    lib.check_status()
    assert bool(torch.isfinite(got).all())
    _check_rows(got[:n], torch.cat(want), BF)
