"""Zosipel's serving kernels beside the like kernels of the closest models (Fedolorn: attention, experts; Zadepel: latent attention; Llama:
decode attention, rotation, projections; Mixtral: routing) at equal sizes: ``python -m levanter_b200.inference.bench_zosipel``, or
``bench.py --mode zosipel``, which adds the engine's prefill and decode throughput.  Timing and rooflines as in ``bench_fedolorn``."""
from __future__ import annotations

import argparse
import json

import torch

from ..ops import lib
from .bench_fedolorn import F32, Table, _pages, _randn


def _difference():
    from ..ops.map_difference import MapDifference

    return MapDifference(torch.full((1,), 0.7, device="cuda"), 0.3, 1e-6)


def attention(tb: Table, T=8192, n_seq=4, H=32, KV=8, S=64, ctx=4096):
    from ..ops import flash_attention as FA
    from ..ops import paged_attention as PA

    diff = _difference()
    L = T // n_seq
    pos = (torch.arange(T, device="cuda") % L).int()

    def seen(window):
        w = min(window or L, L)
        return n_seq * (w * (w + 1) / 2 + (L - w) * w)

    for dk, dv, window, cap in ((64, 128, None, None), (64, 128, None, 30.0), (64, 128, 1024, 30.0), (128, 128, None, None), (32, 64, 256, 30.0)):
        y = _randn(T, 2 * H * dk + KV * (2 * dk + dv) + H)
        q, k = y[:, :2 * H * dk].unflatten(1, (2 * H, dk)), y[:, 2 * H * dk:2 * (H + KV) * dk].unflatten(1, (2 * KV, dk))
        v, gate = y[:, 2 * (H + KV) * dk:-H].unflatten(1, (KV, dv)), y[:, -H:]
        d = 64 if max(2 * dk, dv) <= 64 else 128
        ql, kl, vl = (_randn(T, h, d) for h in (H, KV, KV))
        tb.pair(f"prefill differential 2x{dk}/{dv}, window {window or 'none'}, cap {cap or 'none'}, gated",
                lambda: FA.flash_attention_packed(q, k, v, pos, scaling_factor=dk ** -0.5, window=window, gate=gate, logits_soft_cap=cap, difference=diff),
                f"Fedolorn prefill attention {d}/{d}, window {window or 'none'}, cap {cap or 'none'}",
                lambda: FA.flash_attention_packed(ql, kl, vl, pos, scaling_factor=d ** -0.5, window=window, logits_soft_cap=cap),
                flops=4.0 * H * (dk + dv) * seen(window), nbytes=2.0 * (y.numel() + T * H * dv),
                like_flops=4.0 * H * d * seen(window), like_bytes=4.0 * T * (H + KV) * d)
    sink = _randn(H, dtype=F32)
    for dk, dv in ((128, 128), (64, 64)):
        y = _randn(T, H * (2 * dk + dv))
        q, k, v = (y[:, a:a + H * d].unflatten(1, (H, d)) for a, d in ((0, dk), (H * dk, dk), (2 * H * dk, dv)))
        tb.pair(f"prefill latent {dk}/{dv}, sink", lambda: FA.flash_attention_packed(q, k, v, pos, scaling_factor=dk ** -0.5, sink=sink),
                f"Zadepel prefill latent {dk}/{dv}", lambda: FA.flash_attention_packed(q, k, v, pos, scaling_factor=dk ** -0.5),
                flops=2.0 * H * (dk + dv) * seen(None), nbytes=2.0 * (y.numel() + T * H * dv))

    for dk, dv, window, cap, seqs in ((64, 128, None, None, S), (64, 128, None, 30.0, S), (64, 128, 1024, 30.0, S), (64, 128, None, 30.0, 8), (32, 64, None, 30.0, S)):
        kv, b = _pages(seqs, ctx - 1, 16, KV, 2 * dk + dv)
        q, gate = _randn(seqs, 2 * H, dk), _randn(seqs, H)
        n = min(window or ctx, ctx)
        d = 64 if dv == 64 else 128
        kvl, bl = _pages(seqs, ctx - 1, 16, KV, 2 * d)
        ql2 = _randn(seqs, H, d)
        tb.pair(f"decode differential 2x{dk}/{dv}, {seqs} x {n} keys, cap {cap or 'none'}, gated",
                lambda: PA.paged_attention_general(q, kv, KV, dv, b, sm_scale=dk ** -0.5, window=window, gate=gate, soft_cap=cap, difference=diff),
                f"Fedolorn decode attention {d}/{d}, {seqs} x {n} keys, cap {cap or 'none'}",
                lambda: PA.paged_attention_general(ql2, kvl, KV, d, bl, sm_scale=d ** -0.5, window=window, soft_cap=cap),
                nbytes=2.0 * seqs * (n * KV * (2 * dk + dv) + H * (2 * dk + dv + 1)), like_bytes=2.0 * seqs * (n * KV * 2 * d + 2 * H * d))
    for heads, rank, seqs in ((32, 512, S), (32, 256, S), (16, 512, S), (32, 512, 8)):
        sk = _randn(heads, dtype=F32)
        kv, b = _pages(seqs, ctx - 1, 16, 1, rank)
        kvz, bz = _pages(seqs, ctx - 1, 16, 1, rank + 64)
        q, qz = _randn(seqs, heads, rank), _randn(seqs, heads, rank + 64)
        io = lambda w: dict(flops=2.0 * seqs * ctx * heads * (rank + w), nbytes=2.0 * seqs * (ctx * w + heads * (rank + w)))  # noqa: E731
        tb.pair(f"decode latent, {heads} heads, {rank}, sink, {seqs} x {ctx} keys", lambda: PA.paged_attention_latent(q, kv, rank, b, sm_scale=0.1, sink=sk),
                f"Zadepel decode latent {rank}+64", lambda: PA.paged_attention_latent(qz, kvz, rank, bz, sm_scale=0.1), **io(rank),
                **{"like_" + ("bytes" if n == "nbytes" else n): x for n, x in io(rank + 64).items()})


def around_attention(tb: Table, H=32, KV=8, D=64, Dv=128, rank=512, E=4096):
    from ..layers.rotary import DefaultRotaryEmbeddingsConfig, PartialYarnRotaryEmbeddingsConfig
    from ..ops.norm import rms_norm
    from ..ops.qkv_prep import prepare_latent, prepare_qkv
    from ..ops.residual_stream import project, rms_norm_stream

    rot = PartialYarnRotaryEmbeddingsConfig(theta=500000.0, factor=4.0, original_max_position_embeddings=2048).build(D)
    rotz = DefaultRotaryEmbeddingsConfig().build(2 * D)
    roti = DefaultRotaryEmbeddingsConfig(interleaved=True).build(64)
    wn, wx, add = _randn(rank), _randn(E, scale=0.1), _randn(E)
    whole = _randn(H * 256, rank, scale=0.05)
    n = 2 * H * D + KV * (2 * D + Dv) + H
    wq, bq, wl = _randn(n, E, scale=0.02), _randn(n), _randn(H * 128 + rank, E, scale=0.02)
    n3 = (H + 2 * KV) * 128
    w3 = _randn(n3, E, scale=0.02)
    for T in (64, 8192):
        dest = torch.arange(T, device="cuda", dtype=torch.int32)
        pos = dest % 2048
        y = _randn(T, n)
        q, k = y[:, :2 * H * D].unflatten(1, (2 * H, D)), y[:, 2 * H * D:2 * (H + KV) * D].unflatten(1, (2 * KV, D))
        v = y[:, 2 * (H + KV) * D:-H].unflatten(1, (KV, Dv))
        kv = _randn(T // 16 + 1, 16, KV, 2 * D + Dv)
        qz, kz = y[:, :2 * H * D].unflatten(1, (H, 2 * D)), y[:, 2 * H * D:2 * (H + KV) * D].unflatten(1, (KV, 2 * D))
        tb.pair(f"T={T}: rotate two maps, cache write", lambda: prepare_qkv(q, k, v, kv, dest, pos, rot=rot), "Zadepel rotation and cache write",
                lambda: prepare_qkv(qz, kz, v, kv, dest, pos, rot=rotz), nbytes=2.0 * T * (4 * H * D + KV * (6 * D + 2 * Dv)))
        yl = _randn(T, H * 192 + rank + 64)
        down, downz, qr = yl[:, H * 192:H * 192 + rank], yl[:, H * 192:], yl[:, :H * 192].unflatten(1, (H, 192))[..., 128:]
        pl, plz = _randn(T // 16 + 1, 16, 1, rank), _randn(T // 16 + 1, 16, 1, rank + 64)
        xr = down.contiguous()
        new = lambda: prepare_latent(down, wn, 1e-6, pl, dest, pos, None, qr)  # noqa: E731
        tb.pair(f"T={T}: latent norm, cache write", new, "Zadepel latent norm, rotations, cache write",
                lambda: prepare_latent(downz, wn, 1e-6, plz, dest, pos, roti, qr), nbytes=6.0 * T * rank, like_bytes=2.0 * T * (3 * (rank + 64) + 2 * H * 64))
        tb.pair(f"T={T}: latent norm, cache write (again)", new, f"Llama RMS norm of {rank}", lambda: rms_norm(xr, wn), nbytes=6.0 * T * rank,
                like_bytes=4.0 * T * rank)
        x, h = _randn(T, E, dtype=F32), _randn(T, E)
        tb.pair(f"T={T}: add a vector to the stream, RMS norm", lambda: rms_norm_stream(x, wx, 1e-6, w_offset=1.0, add=add), "Fedolorn RMS norm",
                lambda: rms_norm_stream(x, wx, 1e-6, w_offset=1.0), nbytes=10.0 * T * E, like_bytes=6.0 * T * E)
        g = lambda m, kk, out: dict(flops=2.0 * T * m * kk, nbytes=2.0 * (T * kk + m * kk) + out)  # noqa: E731
        lk = lambda m, kk, out: dict(like_flops=2.0 * T * m * kk, like_bytes=2.0 * (T * kk + m * kk) + out)  # noqa: E731
        tb.pair(f"T={T}: both maps' q and k, v, gate with bias", lambda: project(h, wq, bias=bq), "Llama q, k, v in one product", lambda: project(h, w3),
                **g(n, E, 2.0 * T * n), **lk(n3, E, 2.0 * T * n3))
        nl = wl.shape[0]
        tb.pair(f"T={T}: latent q and down projection", lambda: project(h, wl), "Llama q, k, v in one product", lambda: project(h, w3), **g(nl, E, 2.0 * T * nl),
                **lk(n3, E, 2.0 * T * n3))
        if T > 64:
            lat, nw = _randn(T, rank), whole.shape[0]
            wz = _randn(H * 320, rank + 64, scale=0.05)
            latz = _randn(T, rank + 64)
            tb.pair(f"T={T}: whole keys and values from the latent", lambda: project(lat, whole), "Zadepel whole keys and values", lambda: project(latz, wz),
                    **g(nw, rank, 2.0 * T * nw), **lk(H * 256, rank, 2.0 * T * H * 320))


def experts(tb: Table, E=4096, ff=1024, n=64, k=8, groups=8, keep=4, shared=2048):
    from ..ops import moe
    from ..ops.moe import RoutedTokens
    from ..ops.residual_stream import add_linear, glu_of_rows, project
    from ..utils.activation import ActivationFunctionEnum as A
    from ..models.llama import gated_activation

    gu, down = _randn(n, 2 * ff, E, scale=0.02), _randn(n, E, ff, scale=0.02)
    upf, downf = _randn(n, 3 * ff // 2, E, scale=0.02), _randn(n, E, 3 * ff // 2, scale=0.02)  # as many weights in two matrices
    rows_j = 2 * shared + n + 1
    rows_j += -rows_j % 8
    wj, ws = _randn(rows_j, E, scale=0.02), _randn(E, shared, scale=0.02)
    wu = _randn(2 * shared, E, scale=0.02)
    for T in (8, 64, 256, 8192):
        h, x = _randn(T, E), _randn(T, E, dtype=F32)
        y = _randn(T, rows_j, dtype=F32)
        z, zc = y[:, 2 * shared:2 * shared + n], _randn(T, n, dtype=F32)
        tb.pair(f"T={T}: softmax routing in groups, {n} experts", lambda: moe.route_softmax(z, k, groups=groups, keep=keep), "Fedolorn routing",
                lambda: moe.route_sigmoid(zc, None, k, groups=groups, keep=keep), nbytes=T * (4.0 * n + 8 * k))
        r = moe.route_softmax(z, k, groups=groups, keep=keep)
        used = int((r.counts[:n] > 0).sum())
        counts = r.counts.clone()

        def layer(up, dn, gated):
            counts[n:] = 0
            moe.add_expert_outputs(x, h, RoutedTokens(r.idx, r.w, counts), up, dn, gated=gated)

        rows = moe._block_rows(T * k, n)
        bl = (T * k + min(n, T * k) * (rows - 1) + rows - 1) // rows
        tile = torch.full((bl,), -1, dtype=torch.int32, device="cuda")
        per = (r.counts[:n].long() + rows - 1) // rows
        tile[:int(per.sum())] = torch.repeat_interleave(torch.arange(n, device="cuda"), per).int()
        a, a1, a2 = _randn(bl * rows, E), _randn(bl * rows, ff), _randn(bl * rows, 3 * ff // 2)
        fl = lambda m: dict(flops=2.0 * T * k * m * E, nbytes=2.0 * used * m * E + 2.0 * T * k * (E + m))  # noqa: E731
        lk = lambda m: {"like_" + ("bytes" if key == "nbytes" else key): v for key, v in fl(m).items()}  # noqa: E731
        tb.pair(f"T={T}: expert gate and up product, {used} experts in blocks of {rows}", lambda: moe.grouped_product(a, gu, tile, rows, False),
                "Fedolorn expert up product", lambda: moe.grouped_product(a, upf, tile, rows, True), **fl(2 * ff), **lk(3 * ff // 2))
        tb.pair(f"T={T}: expert down product", lambda: moe.grouped_product(a1, down, tile, rows, False), "Fedolorn expert down product",
                lambda: moe.grouped_product(a2, downf, tile, rows, False), **fl(ff), **lk(3 * ff // 2))
        tb.pair(f"T={T}: whole expert layer after routing (dispatch, products, activation, combine)", lambda: layer(gu, down, True), "Fedolorn expert layer",
                lambda: layer(upf, downf, False), flops=6.0 * T * k * ff * E, nbytes=6.0 * used * ff * E + 8.0 * T * E)
        g = lambda m, kk, out: dict(flops=2.0 * T * m * kk, nbytes=2.0 * (T * kk + m * kk) + out)  # noqa: E731
        tb.pair(f"T={T}: shared gate and up, router in one product, fp32", lambda: project(h, wj, out_dtype=F32), "Zadepel gate and up in one product",
                lambda: project(h, wu), **g(rows_j, E, 4.0 * T * rows_j), like_flops=4.0 * T * shared * E, like_bytes=2.0 * (T * E + 2 * shared * E + 2 * T * shared))
        b16 = y.to(torch.bfloat16)
        tb.pair(f"T={T}: shared silu gate times the token's number", lambda: glu_of_rows(y, shared, A.silu, gate_logit=y[:, 2 * shared + n], out_dtype=torch.bfloat16),
                "Llama silu gate", lambda: gated_activation(b16[:, :shared], b16[:, shared:2 * shared], A.silu), nbytes=10.0 * T * shared, like_bytes=6.0 * T * shared)
        act = _randn(T, shared)
        tb.pair(f"T={T}: shared down product + fp32 stream", lambda: add_linear(x, act, ws), **g(E, shared, 8.0 * T * E))


def kernel_table() -> dict:
    tb = Table()
    with torch.no_grad():
        for part in (attention, around_attention, experts):
            part(tb)
            torch.cuda.empty_cache()
    lib.check_status()
    return {"peaks": {"bf16_tflops": tb.tflops, "hbm_gbs": tb.gbs, "source": tb.how}, "kernels": tb.rows,
            "largest_distance": max(r.get("distance", 0.0) for r in tb.rows)}


def main(argv=None):
    argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter).parse_args(argv)
    out = kernel_table()
    for r in out["kernels"]:
        print(json.dumps(r))
    print(json.dumps({k: v for k, v in out.items() if k != "kernels"}))


if __name__ == "__main__":
    main()
