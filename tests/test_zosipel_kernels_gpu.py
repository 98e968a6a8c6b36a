"""The kernels Zosipel serves with, one mechanism at a time, against the plain statement in ``zosipel_oracle``."""
import pytest
import torch

import zosipel_oracle as O
from levanter_b200.layers.rotary import PartialYarnRotaryEmbeddingsConfig
from levanter_b200.ops import lib
from levanter_b200.ops.map_difference import MapDifference, difference_weight
from levanter_b200.utils.activation import ActivationFunctionEnum
from test_zadepel_kernels_gpu import BF, F32, _check_rows, _randn, _rel, _Sequences

pytestmark = pytest.mark.gpu


def _difference(lam, diff, eps):
    return MapDifference(torch.tensor([lam], device="cuda"), 1.0 - diff, eps)


def _map_needles(q, k, border):
    """``q [n, H, 2, d]``, ``k [n, G, 2, d]``: around every border, one key that stands out for the queries near it in one map, the next
    border's in the other: a mask that is one position off, or a map that reads the other's keys, gives those rows another value."""
    n, d = q.shape[0], q.shape[3]
    for i, b in enumerate(range(border, n, max(border, 3))):
        for key in (b - border, b - border + 1):
            c = key % d
            k[key, :, i % 2] = 0.0
            k[key, :, i % 2, c] = 12.0 if key == b - border else 10.0
            q[max(0, b - 1):b + 2, :, i % 2, c] += 6.0


def test_difference():
    v = [_randn(33, seed=i, dtype=F32, scale=0.4) for i in range(4)]
    w = difference_weight(*(t.cuda() for t in v), 0.35)
    want = O.difference_weight(*(t.double() for t in v), 0.35)
    assert w.shape == (1,) and abs(float(w) - float(want)) < 1e-6
    a, b = _randn(5, 3, 40, seed=7), _randn(5, 3, 40, seed=8)
    got = MapDifference(w, 0.65, 0.02)(a.cuda(), b.cuda())
    assert _rel(got, O.rms(a.double() - want * b.double(), 0.02) * 0.65) < 1e-6


# ------------------------------------------------------------------------------------------------ around attention
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("H,KV,dk,dv,dims,yarn", [(4, 2, 48, 40, 32, (4.0, 30, 8.0, 1.0)), (3, 1, 22, 10, 6, (2.0, 9, 4.0, 2.0)), (2, 2, 64, 128, 64, None),
                                                  (5, 5, 16, 8, 16, (8.0, 100, 32.0, 0.5))])
def test_prepare_two_maps(dtype, H, KV, dk, dv, dims, yarn):
    """Both maps of q and k turn; a slot of the cache holds both keys of a head side by side and then its value."""
    from levanter_b200.ops.qkv_prep import prepare_qkv

    seqs = _Sequences(3, page=4)
    seqs.step([(0, 3), (1, 9)])
    b, pos = seqs.step([(1, 4), (0, 1), (2, 6)])
    T = pos.shape[0]
    wide = _randn(T, 2 * (H + KV) * dk + KV * dv + 8, dtype=dtype).cuda()
    q, k, v = (wide[:, a:a + h * d].unflatten(1, (h, d)) for a, h, d in ((0, 2 * H, dk), (2 * H * dk, 2 * KV, dk), (2 * (H + KV) * dk, KV, dv)))
    ref = dict(base=300.0, dims=dims)
    kw = {}
    if yarn is not None:
        ref["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
        kw = dict(factor=yarn[0], original_max_position_embeddings=yarn[1], beta_fast=yarn[2], beta_slow=yarn[3])
    rot = PartialYarnRotaryEmbeddingsConfig(theta=300.0, rotary_dim=dims, **kw).build(dk)
    q0, k0, v0 = (t.double().cpu() for t in (q, k, v))
    kv = torch.full((160, 4, KV, 2 * dk + dv), 7.0, dtype=dtype, device="cuda")
    with torch.no_grad():
        q, k, v = prepare_qkv(q, k, v, kv, b.new_token_dests, pos, rot=rot)
    at = 0
    for n, start in ((4, 9), (1, 3), (6, 0)):
        rows = slice(at, at + n)
        q0[rows], k0[rows] = O.rotate(q0[rows], ref, start), O.rotate(k0[rows], ref, start)
        at += n
    for got, want in ((q, q0), (k, k0), (v, v0)):
        assert _rel(got[:at], want[:at]) < (1e-6 if dtype == F32 else 4e-3)
    flat, dest = kv.view(-1, KV, 2 * dk + dv), b.new_token_dests[:at].long()
    assert torch.equal(flat[dest], torch.cat([k[:at].reshape(at, KV, 2 * dk), v[:at]], dim=-1))
    assert int((flat != 7.0).any(dim=-1).any(dim=-1).sum()) == at  # nothing else was written


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("rank,H,dn", [(72, 6, 40), (50, 3, 10), (520, 1, 8), (1536, 2, 16), (256, 4, 24)])
def test_prepare_latent_without_positions(dtype, rank, H, dn):
    from levanter_b200.ops.qkv_prep import prepare_latent

    seqs = _Sequences(2, page=4)
    seqs.step([(1, 5)])
    b, pos = seqs.step([(0, 7), (1, 2)])
    T = pos.shape[0]
    wide = _randn(T, H * dn + rank + 8, dtype=dtype, scale=2.0).cuda()
    q, down = wide[:, :H * dn].unflatten(1, (H, dn)), wide[:, H * dn:H * dn + rank]
    w = _randn(rank, seed=3, dtype=dtype)
    kv = torch.full((160, 4, 1, rank), 7.0, dtype=dtype, device="cuda")
    before = q.clone()
    with torch.no_grad():
        latent, _ = prepare_latent(down, w.cuda(), 0.02, kv, b.new_token_dests, pos, None, q[..., dn:])
        kv2 = torch.full_like(kv, 7.0)
        prepare_latent(down, w.cuda(), 0.02, kv2, b.new_token_dests, pos, None, q[..., dn:], to_cache_only=True)
    want = O.rms(down[:9].double().cpu(), 0.02) * w.double()
    assert _rel(latent[:9], want) < (2e-6 if dtype == F32 else 4e-3) and torch.equal(q, before) and torch.equal(kv, kv2)
    flat = kv.view(-1, rank)
    assert torch.equal(flat[b.new_token_dests[:9].long()], latent[:9]) and int((flat != 7.0).any(dim=-1).sum()) == 9


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("dim", [336, 50, 4096])
def test_norm_after_adding_a_vector(dtype, dim):
    from levanter_b200.ops.residual_stream import rms_norm_stream

    x = _randn(7, dim, dtype=F32)
    step, w = _randn(3, dim, seed=1, dtype=dtype), _randn(dim, seed=2, dtype=dtype, scale=0.3)
    want = x.double() + step[1].double()
    with torch.no_grad():
        xc = x.cuda()
        h = rms_norm_stream(xc, w.cuda(), 0.03, w_offset=1.0, add=step.cuda()[1])
    assert _rel(xc, want) < 1e-7 and h.dtype == dtype and _rel(h, O.offset_rms_norm(want, w.double(), 0.03)) < (3e-7 if dtype == F32 else 3e-3)


@pytest.mark.parametrize("y_dtype,out,cols", [(F32, BF, 72), (F32, BF, 30), (F32, F32, 64), (F32, F32, 21), (BF, BF, 40), (BF, BF, 14)])
@pytest.mark.parametrize("gated", [True, False])
def test_silu_gate_times_a_number_per_row(y_dtype, out, cols, gated):
    from levanter_b200.ops.residual_stream import glu_of_rows

    y = _randn(37, 2 * cols + 5, dtype=y_dtype, scale=2.0)
    s = _randn(37, 3, seed=1, dtype=F32, scale=2.0)
    with torch.no_grad():
        got = glu_of_rows(y.cuda(), cols, ActivationFunctionEnum.silu, gate_logit=s.cuda()[:, 1] if gated else None, out_dtype=out)
    want = O.silu(y[:, :cols].double()) * y[:, cols:2 * cols].double()
    if gated:
        want = want * O.sigmoid(s[:, 1:2].double())
    assert got.dtype == out and _rel(got, want) < (1e-6 if out == F32 else 5e-3)


# ------------------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("E,k,groups,keep", [(12, 3, 4, 2), (64, 8, 8, 4), (7, 7, 1, 1), (10, 2, 5, 5), (1, 1, 1, 1), (160, 6, 4, 1), (6, 1, 6, 3)])
def test_softmax_routing_in_groups(E, k, groups, keep):
    from levanter_b200.ops.moe import route_softmax, route_softmax_reference

    wide = _randn(70, E + 5, dtype=F32, scale=3.0).cuda()
    z = wide[:, 2:2 + E]  # strided rows
    live = torch.arange(70, dtype=torch.int32, device="cuda")
    live[5], live[9] = -1, 2_000_000
    r = route_softmax(z, k, groups=groups, keep=keep, live=live, live_limit=1000)
    idx, w = O.route(z.double().cpu(), k, groups, keep)
    ok = torch.ones(70, dtype=torch.bool)
    ok[[5, 9]] = False
    assert torch.equal(r.idx.cpu()[ok].long(), idx[ok]) and bool((r.idx.cpu()[~ok] == -1).all()) and bool((r.w.cpu()[~ok] == 0).all())
    assert float((r.w.cpu().double() - w)[ok].abs().max()) < 1e-6
    assert torch.equal(r.counts[:E].cpu().long(), torch.bincount(idx[ok].reshape(-1), minlength=E))
    i2, w2 = route_softmax_reference(z, k, groups, keep)
    assert torch.equal(i2.cpu(), idx) and float((w2.cpu().double() - w).abs().max()) < 1e-6


@pytest.mark.parametrize("dtype,width,ff,E", [(BF, 352, 72, 14), (BF, 72, 136, 6), (BF, 50, 30, 5), (F32, 96, 40, 7), (BF, 512, 384, 3)])
@pytest.mark.parametrize("T,k", [(1, 2), (9, 3), (150, 2), (700, 3)])
def test_gated_expert_outputs(dtype, width, ff, E, T, k):
    from levanter_b200.ops.moe import add_expert_outputs, expert_outputs, route_softmax

    h, gu = _randn(T, width, dtype=dtype), _randn(E, 2 * ff, width, seed=1, dtype=dtype, scale=width ** -0.5)
    down, x = _randn(E, width, ff, seed=2, dtype=dtype, scale=ff ** -0.5), _randn(T, width, seed=3, dtype=F32)
    z = _randn(T, E, seed=4, dtype=F32)
    z[: T // 2, 1] += 6.0  # a crowded expert
    with torch.no_grad():
        r = route_softmax(z.cuda(), k)
        got = add_expert_outputs(x.cuda(), h.cuda(), r, gu.cuda(), down.cuda(), gated=True)
    lib.check_status()
    idx, w = O.route(z.double(), k, 1, 1)
    want = torch.zeros(T, width, dtype=torch.float64)
    for e in range(E):
        y = O.gated_feed_forward(h.double(), gu[e, :ff].double(), gu[e, ff:].double(), down[e].double())
        for j in range(k):
            m = idx[:, j] == e
            want[m] += w[m, j][:, None] * y[m]
    assert _rel(got.cpu().double() - x.double(), want) < (1e-6 if dtype == F32 else 1e-2)
    diff = expert_outputs(h.cuda(), r.idx, r.w, gu.cuda(), down.cuda(), gated=True)  # the differentiable form agrees
    assert _rel(diff, want) < (1e-6 if dtype == F32 else 1e-2)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("width,ff,E,k,groups,keep,shared", [(72, 24, 10, 3, 5, 2, 40), (64, 16, 6, 2, 1, 1, None), (50, 10, 6, 2, 3, 2, 22), (136, 40, 8, 8, 2, 2, 56)])
def test_mixture_with_shared_expert(dtype, width, ff, E, k, groups, keep, shared):
    """The whole layer on the joint product, for few and many tokens."""
    from levanter_b200.layers.experts import GroupedSoftmaxMoe

    torch.manual_seed(0)
    m = GroupedSoftmaxMoe(width, ff, E, k, groups=groups, keep=keep, shared_intermediate=shared, init_std=0.3).to("cuda", dtype).eval()
    W = {"router": m.router.weight}
    for e in range(E):
        W[f"e{e}.gate"], W[f"e{e}.up"], W[f"e{e}.down"] = m.experts.gate_up[e, :ff], m.experts.gate_up[e, ff:], m.experts.down[e]
    f = dict(router=dict(experts=E, top=k, groups={"count": groups, "keep": keep}))
    if shared is not None:
        f["shared"] = {"ff": shared}
        W.update({"shared.gate": m.shared.gate_proj.weight, "shared.up": m.shared.up_proj.weight, "shared.down": m.shared.down_proj.weight,
                  "shared.sg": m.shared_gate.weight})
    W = {n: t.detach().double().cpu() for n, t in W.items()}
    for T in (3, 300):
        h, x = _randn(T, width, dtype=dtype, seed=T), _randn(T, width, dtype=F32, seed=T + 1)
        want = x.double() + O.mixture_of_experts(h.double(), f, W, "")
        with torch.no_grad():
            got = m.add_to_stream(x.cuda(), h.cuda())
        lib.check_status()
        err = (got.double().cpu() - want).pow(2).mean(-1).sqrt() / (want - x.double()).pow(2).mean().sqrt()
        if dtype == F32:
            assert float(err.max()) < 1e-5
        else:  # a close call of the router may go another way
            assert float(err.median()) < 0.01 and float((err > 0.05).double().mean()) < 0.02


# ------------------------------------------------------------------------------------------------ attention
DIFFERENTIAL = [(BF, 4, 2, 48, 88, 100, 4.0), (BF, 4, 1, 64, 128, None, 30.0), (BF, 2, 2, 32, 64, 48, None), (BF, 8, 1, 128, 256, 300, 20.0),
                (BF, 6, 3, 40, 72, 7, 2.0), (BF, 2, 1, 16, 8, 1, None), (BF, 18, 2, 24, 40, 50, 5.0), (BF, 3, 3, 10, 18, 33, 3.0), (BF, 4, 2, 96, 64, None, None),
                (BF, 2, 1, 136, 64, 60, None), (F32, 4, 2, 48, 88, 100, 4.0), (F32, 3, 3, 11, 17, None, None), (BF, 16, 2, 64, 128, 600, 10.0),
                (BF, 5, 5, 64, 64, 5000, 8.0)]


@pytest.mark.parametrize("dtype,H,G,dk,dv,window,cap", DIFFERENTIAL)
def test_paged_differential_attention(dtype, H, G, dk, dv, window, cap):
    """Decode rows and portions over pages that hold both maps' keys; window and page borders, far keys, one partition and several."""
    from levanter_b200.ops import paged_attention as PA

    wide = window is None or window > 400
    lens = [1, 2, 401, 33, 300 if wide else window, 32 if wide else window + 1, 700]
    last = [1, 2, 1, 5, 1, 1, 3]
    seqs = _Sequences(len(lens))
    kv = torch.full((160, 16, G, 2 * dk + dv), float("nan"), dtype=dtype, device="cuda")
    data = []
    for i, n in enumerate(lens):
        q, k, v = _randn(n, H, 2, dk, seed=i, dtype=dtype), _randn(n, G, 2, dk, seed=50 + i, dtype=dtype), _randn(n, G, dv, seed=90 + i, dtype=dtype)
        _map_needles(q, k, min(window or 300, 300))  # without a window (or with a wide one): keys far away
        data.append((q, k, v))
        if n > last[i]:
            m = n - last[i]
            b, _ = seqs.step([(i, m)], pad=1)
            PA.kv_page_write_general(kv, torch.cat([k[:m], k[:1]]).flatten(2).cuda(), torch.cat([v[:m], v[:1]]).cuda(), b.new_token_dests)
    b, pos = seqs.step([(i, last[i]) for i in range(len(lens))], pad=2)
    tail = [torch.cat([d[j][-last[i]:] for i, d in enumerate(data)] + [torch.zeros(2, *data[0][j].shape[1:], dtype=dtype)]).cuda() for j in range(3)]
    PA.kv_page_write_general(kv, tail[1].flatten(2), tail[2], b.new_token_dests)
    gate = _randn(sum(last) + 2, H + 3, seed=3, dtype=dtype)
    got = PA.paged_attention_general(tail[0].flatten(1, 2), kv, G, dv, b, sm_scale=0.35, window=window, soft_cap=cap, gate=gate.cuda()[:, 1:1 + H],
                                     difference=_difference(0.7, 0.4, 0.01))
    torch.cuda.synchronize()
    want = torch.cat([O.differential_attention(q.double(), k.double(), v.double(), 0.35, 0.7, 0.4, 0.01, window, cap)[-last[i]:]
                      for i, (q, k, v) in enumerate(data)])
    want = O.gate_heads(want, gate[:-2, 1:1 + H].double())
    assert bool((got[-2:] == 0).all())
    _check_rows(got[:-2], want, dtype)


@pytest.mark.parametrize("H,G,dk,dv,window,cap", [(4, 2, 48, 88, 180, 4.0), (2, 1, 64, 128, None, 30.0), (2, 2, 128, 128, 128, None), (4, 1, 40, 72, 7, 2.0),
                                                  (3, 3, 8, 16, 1, None), (2, 2, 96, 64, 256, 10.0), (4, 4, 32, 64, 31, None), (2, 1, 104, 8, 600, 6.0)])
@pytest.mark.parametrize("gates", ["head", "element", None])
def test_packed_differential_prefill(H, G, dk, dv, window, cap, gates):
    from levanter_b200.ops import flash_attention as FA

    lens = [1, 130, 700, 2, 257]
    n = sum(lens)
    T = -(-n // 256) * 256
    cols = [2 * H * dk, 2 * G * dk, G * dv, H * dv, -H % 8 + H]
    wide = torch.zeros(T, sum(cols), dtype=BF)
    pos = torch.zeros(T, dtype=torch.int32)
    gate = _randn(n, cols[3] + cols[4], seed=11)
    at, want = 0, []
    for i, m in enumerate(lens):
        q, k, v = _randn(m, H, 2, dk, seed=i), _randn(m, G, 2, dk, seed=30 + i), _randn(m, G, dv, seed=60 + i)
        _map_needles(q, k, min(window or 300, 300))
        wide[at:at + m] = torch.cat([q.flatten(1), k.flatten(1), v.flatten(1), gate[at:at + m]], dim=1)
        pos[at:at + m] = torch.arange(m)
        want.append(O.differential_attention(q.double(), k.double(), v.double(), 0.35, 0.6, 0.25, 0.02, window, cap))
        at += m
    want = torch.cat(want)
    q, k, v, ge, gh = wide.cuda().split(cols, dim=1)
    q, k, v = q.unflatten(1, (2 * H, dk)), k.unflatten(1, (2 * G, dk)), v.unflatten(1, (G, dv))
    assert FA.packed_supported(q, k, v, 0.35, 2)
    g = None
    if gates == "head":
        g, want = gh[:, :H], O.gate_heads(want, gate[:, cols[3]:cols[3] + H].double())
    elif gates == "element":
        g, want = ge, want * O.sigmoid(gate[:, :cols[3]].double()).view(n, H, dv)
    got = FA.flash_attention_packed(q, k, v, pos.cuda(), scaling_factor=0.35, window=window, logits_soft_cap=cap, gate=g, difference=_difference(0.6, 0.25, 0.02))
    torch.cuda.synchronize()
    lib.check_status()
    assert bool(torch.isfinite(got).all())
    _check_rows(got[:n], want, BF)


def test_gate_per_head_and_soft_cap_with_one_map():
    """The other forms of attention take the gate per head too; the soft cap is exact to bf16 whatever the scores' size."""
    from levanter_b200.ops import flash_attention as FA
    from levanter_b200.ops import paged_attention as PA

    H, G, dk, dv, n = 4, 2, 64, 128, 256
    q, k, v, gate = _randn(n, H, dk), _randn(n, G, dk, seed=1), _randn(n, G, dv, seed=2), _randn(n, H, seed=3)
    seqs = _Sequences(1)
    b, pos = seqs.step([(0, n)], pad=0)
    kv = torch.zeros(160, 16, G, dk + dv, dtype=BF, device="cuda")
    PA.kv_page_write_general(kv, k.cuda(), v.cuda(), b.new_token_dests)
    for scale, cap in ((0.02, 1.0), (0.5, 3.0), (2.0, 50.0)):
        want = torch.stack([O.attend(q[:, h].double(), k[:, h // 2].double(), v[:, h // 2].double(), scale, None, cap) for h in range(H)], dim=1)
        want = O.gate_heads(want, gate.double())
        kw = dict(gate=gate.cuda())
        packed = FA.flash_attention_packed(q.cuda(), k.cuda(), v.cuda(), pos, scaling_factor=scale, logits_soft_cap=cap, **kw)
        paged = PA.paged_attention_general(q.cuda(), kv, G, dv, b, sm_scale=scale, soft_cap=cap, **kw)
        _check_rows(packed, want, BF)
        _check_rows(paged, want, BF)


LATENT = [(BF, 8, 72, 16), (BF, 16, 128, 16), (BF, 5, 512, 16), (BF, 32, 512, 16), (BF, 33, 256, 8), (BF, 40, 64, 4), (BF, 3, 520, 16), (BF, 4, 50, 16), (F32, 6, 72, 16),
          (F32, 2, 33, 3), (BF, 1, 16, 16), (BF, 6, 384, 64), (BF, 2, 8, 32)]


@pytest.mark.parametrize("dtype,H,rank,page", LATENT)
def test_latent_attention_with_sinks(dtype, H, rank, page):
    """All heads read one row per key, which is also the value; sinks from negligible to far above every score; decode rows and portions."""
    from levanter_b200.ops import paged_attention as PA

    lens = [1, 2, 601, 33, 300, 64, 1000]
    last = [1, 2, 1, 30, 1, 1, 1]
    seqs = _Sequences(len(lens), page=page, pages=2800 // page, per_seq=1024 // page)
    kv = torch.full((2800 // page, page, 1, rank), float("nan"), dtype=dtype, device="cuda")
    flat = kv.view(-1, rank)
    sink = torch.linspace(-30.0, 12.0, H)
    sink[-1] = 300.0 if H > 4 else 2.0
    data = []
    for i, n in enumerate(lens):
        q, k = _randn(n, H, rank, seed=i, dtype=dtype), _randn(n, rank, seed=50 + i, dtype=dtype)
        k[n // 3], q[-1] = 0.0, q[-1] * 0.1  # one far key that stands out for the last row
        k[n // 3, 1], q[-1, :, 1] = 9.0, 9.0
        data.append((q, k))
        if n > last[i]:
            b, _ = seqs.step([(i, n - last[i])], pad=0)
            flat[b.new_token_dests.long()] = k[:n - last[i]].cuda()
    b, pos = seqs.step([(i, last[i]) for i in range(len(lens))], pad=2)
    qt = torch.cat([q[-last[i]:] for i, (q, _) in enumerate(data)] + [torch.zeros(2, H, rank, dtype=dtype)]).cuda()
    flat[b.new_token_dests[:-2].long()] = torch.cat([k[-last[i]:] for i, (_, k) in enumerate(data)]).cuda()
    got = PA.paged_attention_latent(qt, kv, rank, b, sm_scale=0.15, sink=sink.cuda())
    torch.cuda.synchronize()
    lib.check_status()
    want = torch.cat([torch.stack([O.attend(q[:, h].double(), k.double(), k.double(), 0.15, sink=sink[h].double()) for h in range(H)], dim=1)[-last[i]:]
                      for i, (q, k) in enumerate(data)])
    assert bool((got[-2:] == 0).all()) and bool(torch.isfinite(got).all())
    _check_rows(got[:-2], want, dtype)


@pytest.mark.parametrize("H,dk,dv", [(5, 32, 32), (2, 128, 128), (3, 64, 24), (1, 192, 128), (2, 8, 16)])
def test_packed_prefill_with_sinks(H, dk, dv):
    from levanter_b200.ops import flash_attention as FA

    lens = [1, 130, 400, 2]
    n = sum(lens)
    T = -(-n // 256) * 256
    sink = torch.linspace(-20.0, 9.0, H) if H > 1 else torch.tensor([1.5])
    wide = torch.zeros(T, H * (2 * dk + dv), dtype=BF)
    pos = torch.zeros(T, dtype=torch.int32)
    at, want = 0, []
    for i, m in enumerate(lens):
        q, k, v = _randn(m, H, dk, seed=i), _randn(m, H, dk, seed=30 + i), _randn(m, H, dv, seed=60 + i)
        wide[at:at + m] = torch.cat([q.flatten(1), k.flatten(1), v.flatten(1)], dim=1)
        pos[at:at + m] = torch.arange(m)
        want.append(torch.stack([O.attend(q[:, h].double(), k[:, h].double(), v[:, h].double(), 0.3, sink=sink[h].double()) for h in range(H)], dim=1))
        at += m
    q, k, v = (t.unflatten(1, (H, -1)) for t in wide.cuda().split([H * dk, H * dk, H * dv], dim=1))
    got = FA.flash_attention_packed(q, k, v, pos.cuda(), scaling_factor=0.3, sink=sink.cuda())
    torch.cuda.synchronize()
    lib.check_status()
    assert bool(torch.isfinite(got).all())
    _check_rows(got[:n], torch.cat(want), BF)
