"""The kernels Zadepel serves with, one mechanism at a time, against the plain statement in ``zadepel_oracle``."""
import numpy as np
import pytest
import torch

import zadepel_oracle as O
from levanter_b200.inference.page_table import PageTable
from levanter_b200.layers.rotary import DefaultRotaryEmbeddingsConfig
from levanter_b200.ops import lib
from levanter_b200.utils.activation import ActivationFunctionEnum

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32


def _rel(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return float((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt().clamp_min(1e-9))


def _randn(*shape, seed=0, dtype=BF, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


def _check_rows(got, want, dtype):
    got, want = got.double().cpu(), want.double()
    err = (got - want).abs().amax(dim=tuple(range(1, got.dim())))
    tol = (2e-5 if dtype == F32 else 3e-2) * float(want.abs().max())
    assert float(err.max()) < tol, (int(err.argmax()), float(err.max()), tol)


class _Sequences:
    """Sequences on shuffled pages: ``step(rows)`` describes a batch of the next rows of each (name order), with padding rows."""

    def __init__(self, slots, page=16, pages=160, per_seq=64, seed=0):
        self.table = PageTable.init(pages, slots, page, per_seq)
        order = np.random.default_rng(seed).permutation(slots)
        self.slot = {}
        for i in range(slots):
            self.table, s = self.table.assign_seq_id_to_seq(int(order[i]))
            self.slot[i] = s
        self.at = {i: 0 for i in range(slots)}

    def step(self, rows, pad=3):
        sl, pos = [], []
        for i, n in rows:
            sl += [self.slot[i]] * n
            pos += range(self.at[i], self.at[i] + n)
            self.at[i] += n
        bad = [2_000_000] * pad
        self.table, b = self.table.allocate_for_seq(np.asarray(sl + bad, np.int32), np.asarray(pos + bad, np.int32))
        return b.to("cuda"), torch.tensor(pos + [0] * pad, dtype=torch.int32, device="cuda")

    def free(self, i):
        m = np.zeros(len(self.slot), bool)
        m[self.slot[i]] = True
        self.table = self.table.free_pages_for_finished(m)
        self.table, s = self.table.assign_seq_id_to_seq(self.slot[i])
        self.at[i] = 0


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("dim", [336, 50, 4096, 11000])
def test_add_norm(dtype, dim):
    from levanter_b200.ops.residual_stream import add_norm_stream

    x, y = _randn(7, dim, dtype=F32), _randn(7, dim, seed=1, dtype=F32, scale=3.0)
    w1, w2 = _randn(dim, seed=2, dtype=dtype), _randn(dim, seed=3, dtype=dtype)
    want_x = x.double() + O.rms_norm(y.double(), w1.double(), 0.03)
    want_h = O.rms_norm(want_x, w2.double(), 0.03)
    with torch.no_grad():
        xc = x.cuda()
        last = add_norm_stream(xc, y.cuda(), w1.cuda(), w2.cuda(), 0.03, rows=torch.tensor([6, 0, 6], device="cuda"))
        assert torch.equal(xc.cpu(), x)  # with rows the stream stays
        h = add_norm_stream(xc, y.cuda(), w1.cuda(), w2.cuda(), 0.03)
    tol = 3e-7 if dtype == F32 else 3e-3
    assert h.dtype == dtype and _rel(xc, want_x) < 2e-7 and _rel(h, want_h) < tol and _rel(last, want_h[[6, 0, 6]]) < tol


@pytest.mark.parametrize("dtype,cols", [(BF, 72), (BF, 30), (F32, 64), (F32, 21)])
def test_gated_gelu(dtype, cols):
    from levanter_b200.ops.residual_stream import glu_of_rows

    y = _randn(37, 2 * cols, dtype=dtype, scale=2.0)
    with torch.no_grad():
        got = glu_of_rows(y.cuda(), cols, ActivationFunctionEnum.gelu_new)
    assert _rel(got, O.gelu_tanh(y[:, :cols].double()) * y[:, cols:].double()) < (1e-6 if dtype == F32 else 5e-3)


@pytest.mark.parametrize("M,N,K", [(5, 264, 328), (64, 96, 72), (130, 136, 64), (700, 520, 1032)])
def test_products_with_bias(M, N, K):
    from levanter_b200.ops.residual_stream import project

    h, w, b = _randn(M, K), _randn(N, K, seed=1, scale=K ** -0.5), _randn(N, seed=2)
    with torch.no_grad():
        f, y = project(h.cuda(), w.cuda(), bias=b.cuda(), out_dtype=F32), project(h.cuda(), w.cuda(), bias=b.cuda())
    want = h.double() @ w.double().T + b.double()
    assert f.dtype == F32 and _rel(f, want) < 2e-6 and _rel(y, want) < 4e-3


# ------------------------------------------------------------------------------------------------ before attention
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("H,KV,dk,dv,dims,inter,temps,mixed", [(6, 2, 96, 40, 32, False, True, True), (4, 4, 64, 64, 64, False, True, False),
                                                               (5, 1, 48, 24, 24, True, False, True), (3, 3, 22, 10, 6, False, True, True),
                                                               (2, 1, 40, 8, 40, True, True, True), (2, 2, 32, 16, 0, False, False, True)])
def test_prepare_qkv(dtype, H, KV, dk, dv, dims, inter, temps, mixed):
    from levanter_b200.ops.qkv_prep import prepare_qkv

    seqs = _Sequences(3, page=4)
    seqs.step([(0, 3), (1, 9)])
    b, pos = seqs.step([(1, 4), (0, 1), (2, 6)])
    T = pos.shape[0]
    wide = _randn(T, (H + KV) * dk + KV * dv + 8, dtype=dtype).cuda()
    q, k, v = (wide[:, a:a + h * d].unflatten(1, (h, d)) for a, h, d in ((0, H, dk), (H * dk, KV, dk), ((H + KV) * dk, KV, dv)))
    rot = DefaultRotaryEmbeddingsConfig(theta=300.0, rotary_dim=dims, interleaved=inter).build(dk) if dims else None
    temp, lam = _randn(H, seed=4, dtype=dtype), torch.tensor(0.375, dtype=dtype)
    first = _randn(T, KV * dv + 8, seed=5, dtype=dtype)
    q0, k0, v0 = (t.double().cpu() for t in (q, k, v))
    kv = torch.full((160, 4, KV, dk + dv), 7.0, dtype=dtype, device="cuda")
    with torch.no_grad():
        q, k, v = prepare_qkv(q, k, v, kv, b.new_token_dests, pos, rot=rot, head_scale=temp.cuda() if temps else None,
                              v_first=first.cuda()[:, :KV * dv].unflatten(1, (KV, dv)) if mixed else None, mix=lam.cuda())
    at = 0
    for n, start in ((4, 9), (1, 3), (6, 0)):
        rows = slice(at, at + n)
        if dims:
            q0[rows], k0[rows] = O.rotate(q0[rows], 300.0, dims, inter, start), O.rotate(k0[rows], 300.0, dims, inter, start)
        at += n
    if temps:
        q0 = q0 * temp.double()[:, None]
    if mixed:
        v0 = O.mix_values(v0, first[:, :KV * dv].double().view(T, KV, dv), 0.375)
    tol = 1e-6 if dtype == F32 else 4e-3
    n = at
    for got, want in ((q, q0), (k, k0), (v, v0)):
        assert _rel(got[:n], want[:n]) < tol
    flat, dest = kv.view(-1, KV, dk + dv), b.new_token_dests[:n].long()
    assert torch.equal(flat[dest], torch.cat([k[:n], v[:n]], dim=-1))
    assert int((flat != 7.0).any(dim=-1).any(dim=-1).sum()) == n  # nothing else was written


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("H,rank,r,dn", [(6, 72, 24, 40), (3, 50, 6, 10), (1, 520, 64, 8), (9, 16, 8, 128)])
def test_prepare_latent(dtype, H, rank, r, dn):
    from levanter_b200.ops.qkv_prep import prepare_latent

    seqs = _Sequences(2, page=4)
    seqs.step([(1, 5)])
    b, pos = seqs.step([(0, 7), (1, 2)])
    T = pos.shape[0]
    wide = _randn(T, H * (dn + r) + rank + r, dtype=dtype, scale=2.0).cuda()
    q, down = wide[:, :H * (dn + r)].unflatten(1, (H, dn + r)), wide[:, H * (dn + r):]
    w = _randn(rank, seed=3, dtype=dtype)
    rot = DefaultRotaryEmbeddingsConfig(theta=500.0, interleaved=True).build(r)
    q0, d0 = q.double().cpu(), down.double().cpu()
    kv = torch.full((160, 4, 1, rank + r), 7.0, dtype=dtype, device="cuda")
    qa = torch.zeros(T, H, rank + r, dtype=dtype, device="cuda")
    with torch.no_grad():
        latent, _ = prepare_latent(down, w.cuda(), 0.02, kv, b.new_token_dests, pos, rot, q[..., dn:], qa[..., rank:])
        latent2, _ = prepare_latent(down, w.cuda(), 0.02, kv, b.new_token_dests, pos, rot, q[..., dn:])  # in place
    tol = 2e-6 if dtype == F32 else 4e-3
    for rows, start in ((slice(0, 7), 0), (slice(7, 9), 5)):
        assert _rel(latent[rows, :rank], O.rms_norm(d0[rows, :rank], w.double(), 0.02)) < tol
        assert _rel(latent[rows, rank:], O.rotate(d0[rows, None, rank:], 500.0, r, True, start)[:, 0]) < tol
        assert _rel(qa[rows, :, rank:], O.rotate(q0[rows, :, dn:], 500.0, r, True, start)) < tol
    assert torch.equal(latent, latent2) and torch.equal(qa[..., rank:], q[..., dn:]) and _rel(q[..., :dn], q0[..., :dn]) == 0
    flat = kv.view(-1, rank + r)
    assert torch.equal(flat[b.new_token_dests[:9].long()], latent[:9]) and int((flat != 7.0).any(dim=-1).sum()) == 9


# ------------------------------------------------------------------------------------------------ recurrence
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("width", [40, 33, 264])
def test_min_gru_over_packed_rows(dtype, width):
    """Several sequences through steps of many rows and of one, slots that are taken again, gates from nearly closed to nearly open."""
    from levanter_b200.ops.gated_scan import min_gru_packed

    lens = {0: 400, 1: 3, 2: 65, 3: 1, 4: 129}
    seqs = _Sequences(5, per_seq=40)
    z = {i: _randn(n, width, seed=i, dtype=F32, scale=4.0) - 3.0 for i, n in lens.items()}
    u = {i: _randn(n, width, seed=10 + i, dtype=F32) for i, n in lens.items()}
    g = {i: _randn(n, width, seed=20 + i, dtype=F32) for i, n in lens.items()}
    want = {i: O.min_gru(z[i].double(), u[i].double(), torch.zeros(width, dtype=torch.float64)) * g[i].double() * torch.sigmoid(g[i].double())
            for i in lens}
    state = torch.full((5, width), 1e3, device="cuda")  # what a slot held before must not matter
    steps = [[(0, 200), (2, 64), (4, 1)], [(0, 1), (4, 127), (1, 2)], [(1, 1), (0, 1), (2, 1), (4, 1)], [(3, 1), (0, 198)]]
    for round_ in range(2):
        at = {i: 0 for i in lens}
        for rows in steps:
            b, pos = seqs.step(rows)
            y = torch.full((pos.shape[0], 3 * width + 5), float("nan"))
            r = 0
            for i, n in rows:
                s = slice(at[i], at[i] + n)
                y[r:r + n, :3 * width] = torch.cat([z[i][s], u[i][s], g[i][s]], dim=1)
                r += n
            with torch.no_grad():
                got = min_gru_packed(y.cuda()[:, :3 * width], state, b, dtype)
            assert bool((got[r:] == 0).all())
            r = 0
            for i, n in rows:
                assert _rel(got[r:r + n], want[i][at[i]:at[i] + n]) < (1e-6 if dtype == F32 else 4e-3), (round_, rows, i)
                r += n
                at[i] += n
        for i in lens:
            seqs.free(i)


# ------------------------------------------------------------------------------------------------ attention
def _needles(q, k, border):
    """Around every border, one key that scores far above all others for the queries near it: a mask that is one position off gives
    those rows another value altogether."""
    n, _, dk = q.shape
    for b in range(border, n, max(border, 3)):
        for key in (b - border, b - border + 1):
            d = key % dk
            k[key] = 0.0
            k[key, :, d] = 12.0 if key == b - border else 10.0
            q[max(0, b - 1):b + 2, :, d] += 6.0


WINDOWED = [(BF, 6, 3, 96, 88, 180), (BF, 8, 2, 64, 64, 48), (BF, 4, 1, 128, 128, 300), (BF, 4, 4, 40, 72, 7), (BF, 2, 1, 200, 88, 1), (BF, 2, 2, 20, 12, 33),
            (BF, 20, 1, 64, 64, 50), (F32, 6, 2, 104, 80, 170), (F32, 3, 3, 33, 17, 10), (BF, 4, 2, 64, 64, 5000), (BF, 8, 2, 96, 32, None)]


@pytest.mark.parametrize("dtype,H,G,dk,dv,window", WINDOWED)
def test_paged_attention_in_a_window(dtype, H, G, dk, dv, window):
    from levanter_b200.ops import paged_attention as PA

    lens = [1, 2, 401, 33, 300 if window is None or window > 400 else window, 32 if window is None or window > 400 else window + 1]
    last = [1, 2, 1, 5, 1, 1]
    seqs = _Sequences(len(lens))
    kv = torch.full((160, 16, G, dk + dv), float("nan"), dtype=dtype, device="cuda")
    data = []
    for i, n in enumerate(lens):
        q, k, v = _randn(n, H, dk, seed=i, dtype=dtype), _randn(n, G, dk, seed=50 + i, dtype=dtype), _randn(n, G, dv, seed=90 + i, dtype=dtype)
        _needles(q, k, min(window or 300, 300))  # without a window (or with a wide one): keys far away
        data.append((q, k, v))
        if n > last[i]:
            b, _ = seqs.step([(i, n - last[i])], pad=1)
            m = n - last[i]
            PA.kv_page_write_general(kv, torch.cat([k[:m], k[:1]]).cuda(), torch.cat([v[:m], v[:1]]).cuda(), b.new_token_dests)
    b, pos = seqs.step([(i, last[i]) for i in range(len(lens))], pad=2)
    tail = [torch.cat([d[j][-last[i]:] for i, d in enumerate(data)] + [torch.zeros(2, *data[0][j].shape[1:], dtype=dtype)]).cuda() for j in range(3)]
    PA.kv_page_write_general(kv, tail[1], tail[2], b.new_token_dests)
    got = PA.paged_attention_general(tail[0], kv, G, dv, b, sm_scale=0.35, window=window)
    torch.cuda.synchronize()
    want = torch.cat([O.softmax_attention(q.double(), k.double(), v.double(), 0.35, window)[-last[i]:] for i, (q, k, v) in enumerate(data)])
    assert bool((got[-2:] == 0).all())
    _check_rows(got[:-2], want, dtype)


LATENT = [(BF, 8, 72, 24, 40, 16), (BF, 16, 128, 32, None, 16), (BF, 5, 512, 64, 100, 16), (BF, 32, 512, 64, None, 16), (BF, 33, 256, 64, 33, 8),
          (BF, 40, 64, 8, 1, 4), (BF, 3, 520, 64, 50, 16), (BF, 4, 50, 6, 30, 16), (F32, 6, 72, 24, 40, 16), (F32, 2, 33, 6, None, 3), (BF, 1, 16, 8, 7, 16),
          (BF, 24, 88, 16, 129, 16), (BF, 2, 8, 8, 64, 32)]


@pytest.mark.parametrize("dtype,H,rank,r,window,page", LATENT)
def test_latent_attention(dtype, H, rank, r, window, page):
    """All heads read one row per key, whose first part is also the value; decode rows, portions, page and window borders."""
    from levanter_b200.ops import paged_attention as PA

    w = rank + r
    lens = [1, 2, 601, 33, 300 if window is None else window, 64 if window is None else window + 1]
    last = [1, 2, 1, 30, 1, 1]
    seqs = _Sequences(len(lens), page=page, pages=2400 // page, per_seq=1024 // page)
    kv = torch.full((2400 // page, page, 1, w), float("nan"), dtype=dtype, device="cuda")
    flat = kv.view(-1, w)
    data = []
    for i, n in enumerate(lens):
        q, k = _randn(n, H, w, seed=i, dtype=dtype), _randn(n, 1, w, seed=50 + i, dtype=dtype)
        _needles(q, k, min(window or 300, 300))  # without a window (or with a wide one): keys far away
        data.append((q, k))
        if n > last[i]:
            b, _ = seqs.step([(i, n - last[i])], pad=0)
            flat[b.new_token_dests.long()] = k[:n - last[i], 0].cuda()
    b, pos = seqs.step([(i, last[i]) for i in range(len(lens))], pad=2)
    qt = torch.cat([q[-last[i]:] for i, (q, _) in enumerate(data)] + [torch.zeros(2, H, w, dtype=dtype)]).cuda()
    flat[b.new_token_dests[:-2].long()] = torch.cat([k[-last[i]:, 0] for i, (_, k) in enumerate(data)]).cuda()
    got = PA.paged_attention_latent(qt, kv, rank, b, sm_scale=0.21, window=window)
    torch.cuda.synchronize()
    want = torch.cat([O.softmax_attention(q.double(), k.double(), k[..., :rank].double(), 0.21, window)[-last[i]:] for i, (q, k) in enumerate(data)])
    assert bool((got[-2:] == 0).all())
    _check_rows(got[:-2], want, dtype)


@pytest.mark.parametrize("dtype,T,H,N,K", [(BF, 1, 3, 64, 40), (BF, 70, 8, 72, 24), (BF, 65, 2, 512, 128), (BF, 9, 5, 128, 512), (BF, 7, 2, 12, 20), (F32, 30, 4, 48, 33)])
def test_head_products(dtype, T, H, N, K):
    from levanter_b200.ops.paged_attention import head_product

    wide = _randn(T, H, K + 16, dtype=dtype)
    both = _randn(H, 2 * K + 8, N, seed=1, dtype=dtype)
    out = torch.zeros(T, H, N + 8, dtype=dtype, device="cuda")
    a, b = wide.cuda()[..., 8:8 + K], both.cuda()[:, 8:8 + K]
    head_product(a, b, out[..., :N], b_trans=False)
    want = torch.einsum("thk,hkn->thn", wide[..., 8:8 + K].double(), both[:, 8:8 + K].double())
    tol = 1e-6 if dtype == F32 else 4e-3
    assert _rel(out[..., :N], want) < tol and bool((out[..., N:] == 0).all())
    bt = _randn(H, N + 4, K, seed=2, dtype=dtype)
    got = head_product(a, bt.cuda()[:, :N], out.new_zeros(T, H, N), b_trans=True)
    assert _rel(got, torch.einsum("thk,hnk->thn", wide[..., 8:8 + K].double(), bt[:, :N].double())) < tol


@pytest.mark.parametrize("H,G,dk,dv,window", [(6, 3, 96, 88, 180), (2, 1, 64, 64, 128), (2, 2, 128, 128, None), (4, 1, 40, 72, 7), (2, 2, 128, 64, 256),
                                              (3, 3, 8, 16, 1), (2, 2, 192, 128, 200), (2, 2, 136, 24, None), (4, 4, 160, 128, 31), (2, 1, 192, 64, 600)])
def test_packed_prefill_in_a_window(H, G, dk, dv, window):
    from levanter_b200.ops import flash_attention as FA

    lens = [1, 130, 700, 2, 257]
    n = sum(lens)
    T = -(-n // 256) * 256
    wide = torch.zeros(T, (H + G) * dk + G * dv, dtype=BF)
    pos = torch.zeros(T, dtype=torch.int32)
    at, want = 0, []
    for i, m in enumerate(lens):
        q, k, v = _randn(m, H, dk, seed=i), _randn(m, G, dk, seed=30 + i), _randn(m, G, dv, seed=60 + i)
        _needles(q, k, min(window or 300, 300))  # without a window (or with a wide one): keys far away
        wide[at:at + m] = torch.cat([q.flatten(1), k.flatten(1), v.flatten(1)], dim=1)
        pos[at:at + m] = torch.arange(m)
        want.append(O.softmax_attention(q.double(), k.double(), v.double(), 0.35, window))
        at += m
    w = wide.cuda()
    q, k, v = (w[:, a:a + h * d].unflatten(1, (h, d)) for a, h, d in ((0, H, dk), (H * dk, G, dk), ((H + G) * dk, G, dv)))
    assert FA.packed_supported(q, k, v, 0.35)
    got = FA.flash_attention_packed(q, k, v, pos.cuda(), scaling_factor=0.35, window=window)
    torch.cuda.synchronize()
    lib.check_status()
    assert bool(torch.isfinite(got).all())
    _check_rows(got[:n], torch.cat(want), BF)
