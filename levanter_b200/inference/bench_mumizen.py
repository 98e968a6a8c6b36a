"""Mumizen's serving kernels beside the like kernels of the closest models (Zadepel: the recurrence, latent attention, stream norms; Gated
DeltaNet: the scan; Zosipel: experts; Fedolorn and Llama: norms, activations, projections) at equal sizes: ``python -m
levanter_b200.inference.bench_mumizen``, or ``bench.py --mode mumizen``, which adds the engine's prefill and decode throughput.  Timing and
rooflines as in ``bench_fedolorn``."""
from __future__ import annotations

import argparse
import json

import torch

from ..ops import lib
from .bench_fedolorn import BF, F32, Table, _pages, _randn


def _batch(T, n_seq, S):
    """Device tables of ``n_seq`` sequences of ``T / n_seq`` rows each that go on from their slots."""
    L = T // n_seq
    _, b = _pages(S, 1, 16, 1, 8)
    cu = torch.full((S + 1,), T, dtype=torch.int32, device="cuda")
    cu[:n_seq + 1] = torch.arange(n_seq + 1, device="cuda") * L
    b.cu_q_lens, b.num_seqs, b.seq_lens = cu, torch.tensor(n_seq, device="cuda", dtype=torch.int32), torch.full((S,), L + 1, dtype=torch.int32, device="cuda")
    b.longest = L
    return b


def recurrence(tb: Table):
    from ..models.gated_deltanet import delta_rule_chunked_scan
    from ..ops.gated_scan import min_gru_packed
    from ..ops.linear_attention import gated_norm, linear_attention_packed, silu_in_place
    from ..ops.norm import rms_norm

    for T, n_seq, S, H, d in ((8192, 4, 16, 32, 128), (8192, 1, 16, 32, 128), (16384, 16, 16, 32, 128), (8192, 4, 16, 64, 64), (8192, 4, 16, 16, 256), (64, 64, 64, 32, 128), (64, 64, 64, 64, 64),
                              (8, 8, 8, 32, 128)):
        L, W = T // n_seq, H * d
        y = _randn(T, 4 * W)
        q, k, v = (y[:, i * W:(i + 1) * W].unflatten(1, (H, d)) for i in range(3))
        g = torch.linspace(0.6, 0.999, H, device="cuda")
        state, b = torch.zeros(S, H, d, d, device="cuda"), _batch(T, n_seq, S)
        z, zs = _randn(T, 3 * W, dtype=F32), torch.zeros(S, W, device="cuda")
        new = lambda: linear_attention_packed(q, k, v, g, state, b, key_scale=d ** -0.5)  # noqa: E731
        kw = dict(nbytes=8.0 * T * W + 8.0 * n_seq * W * d, flops=4.0 * T * W * d, like_flops=0.0)
        tb.pair(f"linear attention {H} x {d}/{d}, {n_seq} x {L} rows", new, f"Zadepel minGRU of {W}, as many rows", lambda: min_gru_packed(z, zs, b, BF),
                like_bytes=14.0 * T * W + 8.0 * n_seq * W, **kw)
        if L >= 64 and d == 128:
            qd, kd, vd = (_randn(n_seq, H, L, d) for _ in range(3))
            qd, kd = (torch.nn.functional.normalize(t.float(), dim=-1).to(BF) for t in (qd, kd))
            gd, beta = -torch.rand(n_seq, H, L, device="cuda"), torch.rand(n_seq, H, L, device="cuda")
            tb.pair(f"linear attention {H} x {d}/{d}, {n_seq} x {L} rows (again)", new, "Gated DeltaNet scan", lambda: delta_rule_chunked_scan(qd, kd, vd, gd, beta),
                    like_bytes=8.0 * T * W, **kw)
            tb.pair(f"silu of q, k and v, {T} rows of {3 * W}", lambda: silu_in_place(q, k, v), "Llama silu gate", _llama_silu(T, 3 * W // 2), nbytes=12.0 * T * W,
                    like_bytes=9.0 * T * W)
        if d == 128:
            o, gate, w, whole = _randn(T, W), y[:, 3 * W:], _randn(W), _randn(T, W)
            for groups in (1, H):
                tb.pair(f"T={T}: norm of {W} in {groups} groups, gate", lambda: gated_norm(o, gate, 1e-5, groups=groups, weight=w if groups == 1 else None,
                                                                                       sigmoid=groups == 1),
                        f"Llama RMS norm of {W}", lambda: rms_norm(whole, w), nbytes=6.0 * T * W, like_bytes=4.0 * T * W)


def _llama_silu(T, ff):
    from ..models.llama import gated_activation
    from ..utils.activation import ActivationFunctionEnum as A

    y = _randn(T, 2 * ff)
    return lambda: gated_activation(y[:, :ff], y[:, ff:], A.silu)


def stream(tb: Table, E=4096):
    from ..ops.depth_stream import norm_of_depths
    from ..ops.residual_stream import add_norm_stream, rms_norm_stream

    for T, n_seq in ((64, 64), (8192, 4)):
        S = max(n_seq, 16)
        b = _batch(T, n_seq, S)
        hist = _randn(34, T, E, dtype=F32, scale=0.1)
        y, w, mu, w2, state = _randn(T, E, dtype=F32), _randn(E), _randn(E), _randn(E), torch.zeros(S, E, device="cuda")
        like = ("Zadepel norm, add to the stream, norm", lambda: add_norm_stream(hist[0], y, w, w2, 1e-5))
        for planes in (2, 8, 17, 33):
            coef = _randn(planes)
            tb.pair(f"T={T}: average of {planes} depths, norm in 8 groups, token shift",
                    lambda: norm_of_depths(hist[:planes], w, 1e-5, groups=8, coef=coef, out=hist[33], shift=mu, state=state, batch_info=b), *like,
                    nbytes=T * E * (4.0 * planes + 6.0) + 8.0 * n_seq * E, like_bytes=14.0 * T * E)
        tb.pair(f"T={T}: norm in 8 groups", lambda: norm_of_depths(hist[:1], w, 1e-5, groups=8), "Fedolorn RMS norm", lambda: rms_norm_stream(hist[0], w, 1e-5),
                nbytes=6.0 * T * E)


def latent(tb: Table, E=4096, H=32, D=128, R=64, Dv=128, rank=512, q_rank=1536, S=64, ctx=4096):
    from ..layers.rotary import DefaultRotaryEmbeddingsConfig, PartialYarnRotaryEmbeddingsConfig
    from ..ops import flash_attention as FA
    from ..ops import paged_attention as PA
    from ..ops.norm import rms_norm
    from ..ops.qkv_prep import norm_rows, prepare_latent, rotate_queries
    from ..ops.residual_stream import project

    rot = PartialYarnRotaryEmbeddingsConfig(theta=500000.0, factor=4.0, original_max_position_embeddings=2048).build(R)
    roti = DefaultRotaryEmbeddingsConfig(interleaved=True).build(R)
    wn, wq = _randn(rank), _randn(q_rank)
    own, shared, up = q_rank + rank + R + H * Dv, q_rank + H * Dv, H * (D + R)
    w_own, w_shared, w_up, w3 = _randn(own, E, scale=0.02), _randn(shared, E, scale=0.02), _randn(up, q_rank, scale=0.02), _randn(3 * H * D // 2, E, scale=0.02)
    for T in (64, 8192):
        dest = torch.arange(T, device="cuda", dtype=torch.int32)
        pos = dest % 2048
        h, cq = _randn(T, E), _randn(T, q_rank)
        g = lambda m, kk: dict(flops=2.0 * T * m * kk, nbytes=2.0 * (T * kk + m * kk + T * m))  # noqa: E731
        lk = {("like_" + ("bytes" if n == "nbytes" else n)): x for n, x in g(w3.shape[0], E).items()}
        for name, w in (("queries' latent, latent, gate", w_own), ("queries' latent, gate", w_shared)):
            tb.pair(f"T={T}: {name} in one product", lambda: project(h, w), "Llama q, k, v in one product", lambda: project(h, w3), **g(w.shape[0], E), **lk)
        tb.pair(f"T={T}: queries from their latent", lambda: project(cq, w_up), "Llama q, k, v in one product", lambda: project(h, w3), **g(up, q_rank), **lk)
        y = _randn(T, own)
        tb.pair(f"T={T}: norm of the queries' latent", lambda: norm_rows(y[:, :q_rank], wq, 1e-5), f"Llama RMS norm of {q_rank}", lambda: rms_norm(cq, wq),
                nbytes=4.0 * T * q_rank)
        q, down, pages = _randn(T, H, D + R), y[:, q_rank:q_rank + rank + R], _randn(T // 16 + 1, 16, 1, rank + R)
        tb.pair(f"T={T}: latent norm, rotations (halves, YaRN), cache write", lambda: prepare_latent(down, wn, 1e-5, pages, dest, pos, rot, q[..., D:]),
                "Zadepel latent norm, rotations, cache write", lambda: prepare_latent(down, wn, 1e-5, pages, dest, pos, roti, q[..., D:]),
                nbytes=2.0 * T * (3 * (rank + R) + 2 * H * R))
        tb.pair(f"T={T}: rotation of the queries alone", lambda: rotate_queries(q[..., D:], pos, rot), "Zadepel latent norm, rotations, cache write",
                lambda: prepare_latent(down, wn, 1e-5, pages, dest, pos, roti, q[..., D:]), nbytes=4.0 * T * H * R, like_bytes=2.0 * T * (3 * (rank + R) + 2 * H * R))
        o, uv, gate, heads = _randn(T, H, rank), _randn(H, Dv, rank, scale=0.05), y[:, -H * Dv:], torch.empty(T, H, Dv, dtype=BF, device="cuda")
        if T == 64:
            io = dict(flops=2.0 * T * H * Dv * rank, nbytes=2.0 * H * (T * rank + Dv * rank + 2 * T * Dv))
            tb.pair(f"T={T}: heads from the latent, gate", lambda: PA.head_product(o, uv, heads, b_trans=True, gate=gate), "Zadepel heads from the latent",
                    lambda: PA.head_product(o, uv, heads, b_trans=True), **io, like_bytes=2.0 * H * (T * rank + Dv * rank + T * Dv))
        else:
            k, v = _randn(T, H, D + R), _randn(T, H, Dv)
            keys = 4 * 2048 * 2049 / 2
            io = dict(flops=2.0 * H * (D + R + Dv) * keys, nbytes=2.0 * T * H * (2 * (D + R) + 3 * Dv))
            tb.pair(f"prefill latent {D + R}/{Dv}, gated", lambda: FA.flash_attention_packed(q, k, v, pos, scaling_factor=0.07, gate=gate),
                    f"Zadepel prefill latent {D + R}/{Dv}", lambda: FA.flash_attention_packed(q, k, v, pos, scaling_factor=0.07), **io)
    kv, b = _pages(S, ctx - 1, 16, 1, rank + R)
    qz = _randn(S, H, rank + R)
    tb.pair(f"decode latent, {H} heads, {rank}+{R}, {S} x {ctx} keys", lambda: PA.paged_attention_latent(qz, kv, rank, b, sm_scale=0.1),
            flops=2.0 * S * ctx * H * (2 * rank + R), nbytes=2.0 * S * (ctx * (rank + R) + H * (2 * rank + R)))


def feed_forward(tb: Table, E=4096, ff=1024, n=64, k=8, shared=2048, wide=14336):
    from ..ops import moe
    from ..ops.glu import ClampedGlu
    from ..ops.moe import RoutedTokens
    from ..ops.residual_stream import glu_of_rows, project
    from ..utils.activation import ActivationFunctionEnum as A

    act = ClampedGlu(7.0)
    gu, down = _randn(n, 2 * ff, E, scale=0.02), _randn(n, E, ff, scale=0.02)
    rows_j = 2 * shared + n
    wj, wz, bias = _randn(rows_j, E, scale=0.02), _randn(rows_j + 8, E, scale=0.02), _randn(n)
    for T in (8, 64, 8192):
        h, x = _randn(T, E), _randn(T, E, dtype=F32)
        z = _randn(T, n, dtype=F32)
        tb.pair(f"T={T}: softmax routing with a bias, {n} experts", lambda: moe.route_softmax(z, k, bias=bias), "Zosipel routing",
                lambda: moe.route_softmax(z, k, groups=8, keep=4), nbytes=T * (4.0 * n + 8 * k))
        r = moe.route_softmax(z, k, bias=bias)
        used, counts = int((r.counts[:n] > 0).sum()), r.counts.clone()

        def layer(a):
            counts[n:] = 0
            moe.add_expert_outputs(x, h, RoutedTokens(r.idx, r.w, counts), gu, down, gated=True, act=a)

        tb.pair(f"T={T}: expert layer after routing, clamped", lambda: layer(act), "Zosipel expert layer", lambda: layer(A.silu), flops=6.0 * T * k * ff * E,
                nbytes=6.0 * used * ff * E + 8.0 * T * E)
        io = lambda m: dict(flops=2.0 * T * m * E, nbytes=2.0 * (T * E + m * E) + 4.0 * T * m)  # noqa: E731
        tb.pair(f"T={T}: shared gate and up, router in one product, fp32", lambda: project(h, wj, out_dtype=F32), "Zosipel shared gate and up, router, number",
                lambda: project(h, wz, out_dtype=F32), **io(rows_j))
        for cols, dt in ((shared, F32), (wide, BF)):
            y = _randn(T, 2 * cols, dtype=dt)
            like = _llama_silu(T, cols)
            tb.pair(f"T={T}: clamped gate of {cols} from {'fp32' if dt == F32 else 'bf16'}", lambda: glu_of_rows(y, cols, act, out_dtype=BF), "Llama silu gate", like,
                    nbytes=T * cols * (2.0 * y.element_size() + 2.0), like_bytes=6.0 * T * cols)


def kernel_table() -> dict:
    tb = Table()
    with torch.no_grad():
        for part in (recurrence, stream, latent, feed_forward):
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
