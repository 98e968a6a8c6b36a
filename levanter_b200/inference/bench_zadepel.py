"""Zadepel's serving kernels beside the like kernels of the closest models (Llama: attention, rotation, projections, norms; Gated
DeltaNet: the recurrence) at equal sizes: ``python -m levanter_b200.inference.bench_zadepel``, or ``bench.py --mode zadepel``, which
adds the engine's prefill and decode throughput.  Timing and rooflines as in ``bench_fedolorn``."""
from __future__ import annotations

import argparse
import json

import torch

from ..ops import lib
from .bench_fedolorn import BF, F32, Table, _pages, _randn


def attention(tb: Table, T=8192, n_seq=4, H=32, KV=8, S=64, ctx=4096):
    from ..layers.attention import AttentionMask, dot_product_attention
    from ..ops import flash_attention as FA
    from ..ops import paged_attention as PA

    L = T // n_seq
    pos = (torch.arange(T, device="cuda") % L).int()
    seg = (torch.arange(T, device="cuda") // L).int()
    m = AttentionMask.causal().with_segment_ids(seg[None], sorted=True)
    for what, hk, dk, dv, window in (("attention", KV, 128, 128, None), ("attention", KV, 128, 64, None), ("latent", H, 192, 128, None),
                                     ("latent", H, 192, 128, 1024), ("latent", H, 128, 128, 1024), ("latent", H, 96, 64, 256)):
        y = _randn(T, H * dk + hk * (dk + dv))
        q, k, v = (y[:, a:a + h * d].unflatten(1, (h, d)) for a, h, d in ((0, H, dk), (H * dk, hk, dk), ((H + hk) * dk, hk, dv)))
        w = min(window or L, L)
        keys = n_seq * (w * (w + 1) / 2 + (L - w) * w)
        ql, kl, vl = (_randn(1, T, h, 128) for h in (H, hk, hk))
        # Llama prefills with a segment id per key; the packed kernel without a window is the better yardstick, so both are given
        base = dict(flops=2.0 * H * (dk + dv) * keys, nbytes=2.0 * (y.numel() + T * H * dv))
        like = dict(like_flops=4.0 * H * 128 * n_seq * L * (L + 1) / 2, like_bytes=4.0 * T * (H + hk) * 128)
        new = lambda: FA.flash_attention_packed(q, k, v, pos, scaling_factor=dk ** -0.5, window=window)  # noqa: E731
        name = f"prefill {what} {dk}/{dv}, window {window or 'none'}"
        tb.pair(name, new, "Llama prefill attention 128", lambda: dot_product_attention(ql, kl, vl, m), **base, **like)
        if what == "latent":
            tb.pair(name + " (again)", new, "Fedolorn prefill attention 128/128",
                    lambda: FA.flash_attention_packed(ql[0], kl[0], vl[0], pos, scaling_factor=128 ** -0.5), **base, **like)
    def llama_decode(seqs, keys):
        """Llama's decode attention over as many sequences and keys: the call, its name, its bytes."""
        kvl, bl = _pages(seqs, keys - 1, 16, KV, 256)
        kvl = kvl.view(kvl.shape[0], 16, 2 * KV, 128)
        ql = _randn(seqs, H, 128)
        call = lambda: PA.ragged_paged_attention(ql, kvl, bl.seq_lens, bl.page_indices, bl.cu_q_lens, bl.num_seqs, sm_scale=0.1)  # noqa: E731
        return call, f"Llama decode attention 128, {seqs} x {keys} keys", 2.0 * seqs * (keys * KV * 256 + 2 * H * 128)

    for dk, dv in ((128, 128), (128, 64)):
        kv, b = _pages(S, ctx - 1, 16, KV, dk + dv)
        q = _randn(S, H, dk)
        like, like_name, like_bytes = llama_decode(S, ctx)
        tb.pair(f"decode attention {dk}/{dv}, {S} x {ctx} keys", lambda: PA.paged_attention_general(q, kv, KV, dv, b, sm_scale=dk ** -0.5), like_name,
                like, nbytes=2.0 * S * (ctx * KV * (dk + dv) + H * (dk + dv)), like_bytes=like_bytes)
    for heads, rank, r, window, seqs in ((32, 512, 64, None, S), (32, 512, 64, 1024, S), (16, 512, 64, None, S), (32, 256, 32, None, S), (32, 512, 64, None, 8),
                                         (128, 512, 64, None, S)):
        kv, b = _pages(seqs, ctx - 1, 16, 1, rank + r)
        q = _randn(seqs, heads, rank + r)
        seen = min(window or ctx, ctx)
        like, like_name, like_bytes = llama_decode(seqs, seen)
        tb.pair(f"decode latent, {heads} heads, {rank}+{r}, {seqs} x {seen} keys", lambda: PA.paged_attention_latent(q, kv, rank, b, sm_scale=0.1, window=window),
                like_name, like, flops=2.0 * seqs * seen * heads * (2 * rank + r),
                nbytes=2.0 * seqs * (seen * (rank + r) + heads * (2 * rank + r)), like_bytes=like_bytes)


def around_attention(tb: Table, H=32, KV=8, D=128, rank=512, r=64, E=4096):
    from ..layers.rotary import DefaultRotaryEmbeddingsConfig
    from ..ops import paged_attention as PA
    from ..ops.gemm import linear
    from ..ops.qkv_prep import prepare_latent, prepare_qkv
    from ..ops.residual_stream import project
    from ..ops.rope import apply_rope

    rot = DefaultRotaryEmbeddingsConfig(rotary_dim=64).build(D)
    rotl = DefaultRotaryEmbeddingsConfig().build(D)
    roti = DefaultRotaryEmbeddingsConfig(interleaved=True).build(r)
    temp, lam, wn = _randn(H), _randn(1)[0], _randn(rank)
    w = _randn(H, 2 * D, rank, scale=0.05)
    whole = _randn(H * (2 * D + r), rank + r, scale=0.05)
    for T in (64, 8192):
        pages = T // 16 + 1
        dest = torch.arange(T, device="cuda", dtype=torch.int32)
        pos = dest % 2048
        y = _randn(T, (H + 2 * KV) * D)
        q, k, v = (y[:, a:a + h * D].unflatten(1, (h, D)) for a, h in ((0, H), (H * D, KV), ((H + KV) * D, KV)))
        first = _randn(T, KV, D)
        kv, kvl = _randn(pages, 16, KV, 2 * D), _randn(pages, 16, 2 * KV, D)
        ql, kl, vl = _randn(T, H, D), _randn(T, KV, D), _randn(T, KV, D)

        def llama():
            a, b = apply_rope(ql, kl, rotl, pos)
            PA.kv_page_write(kvl, b, vl, dest)
            return a

        llama_bytes = 2.0 * T * D * (2 * H + 2 * KV + 4 * KV)
        tb.pair(f"T={T}: rotate, temper, mix values, cache write", lambda: prepare_qkv(q, k, v, kv, dest, pos, rot=rot, head_scale=temp, v_first=first, mix=lam),
                "Llama rotation and cache write", llama, nbytes=2.0 * T * D * (2 * H + 2 * KV + 3 * KV + 2 * KV), like_bytes=llama_bytes)
        yl = _randn(T, H * (D + r) + rank + r)
        lq, down = yl[:, :H * (D + r)].unflatten(1, (H, D + r)), yl[:, H * (D + r):]
        pl = _randn(pages, 16, 1, rank + r)
        tb.pair(f"T={T}: latent norm, rotations, cache write", lambda: prepare_latent(down, wn, 1e-6, pl, dest, pos, roti, lq[..., D:]),
                "Llama rotation and cache write", llama, nbytes=2.0 * T * (3 * (rank + r) + 2 * H * r), like_bytes=llama_bytes)
        lk = lambda n, kk, out: dict(like_flops=2.0 * T * n * kk, like_bytes=2.0 * (T * kk + n * kk) + out)  # noqa: E731
        if T == 64:
            qa = _randn(T, H, rank + r)
            o = _randn(T, H, rank)
            out = _randn(T, H, D)
            nb = 2.0 * (H * D * rank + T * H * (D + rank))
            ws, as_ = _randn(E, rank, scale=0.02), _randn(T, rank)  # as many weights in one plain product
            small = lambda: linear(as_, ws)  # noqa: E731
            tb.pair(f"T={T}: queries into the latent", lambda: PA.head_product(lq[..., :D], w[:, :D], qa[..., :rank], b_trans=False), f"Llama product {rank} -> {E}",
                    small, flops=2.0 * T * H * D * rank, nbytes=nb, **lk(E, rank, 2.0 * T * E))
            tb.pair(f"T={T}: values out of the latent", lambda: PA.head_product(o, w[:, D:], out, b_trans=True), f"Llama product {rank} -> {E}", small,
                    flops=2.0 * T * H * D * rank, nbytes=nb, **lk(E, rank, 2.0 * T * E))
        else:
            lat = _randn(T, rank + r)
            n = whole.shape[0]
            ws, as_ = _randn(H * 2 * D, rank, scale=0.02), _randn(T, rank)  # the same keys and values without their rotated part
            tb.pair(f"T={T}: whole keys and values from the latent", lambda: project(lat, whole), f"Llama product {rank} -> {H * 2 * D}", lambda: linear(as_, ws),
                    flops=2.0 * T * H * 2 * D * rank, nbytes=2.0 * (T * (rank + r) + H * 2 * D * rank + T * n), **lk(H * 2 * D, rank, 2.0 * T * H * 2 * D))


def recurrence(tb: Table, W=4096):
    from ..models.gated_deltanet import delta_rule_chunked_scan
    from ..ops.gated_scan import min_gru_packed

    for T, n_seq, S in ((8192, 4, 16), (8192, 1, 16), (64, 64, 64)):
        L = T // n_seq
        H = 32
        y = _randn(T, 3 * W, dtype=F32)
        state = torch.zeros(S, W, device="cuda")
        _, b = _pages(S, 1, 16, 1, 8)
        cu = torch.full((S + 1,), T, dtype=torch.int32, device="cuda")
        cu[:n_seq + 1] = torch.arange(n_seq + 1, device="cuda") * L
        b.cu_q_lens, b.num_seqs, b.seq_lens = cu, torch.tensor(n_seq, device="cuda", dtype=torch.int32), torch.full((S,), L + 1, dtype=torch.int32, device="cuda")
        q, k, v = (_randn(n_seq, H, L, W // H) for _ in range(3))
        q, k = (torch.nn.functional.normalize(t.float(), dim=-1).to(BF) for t in (q, k))
        g, beta = -torch.rand(n_seq, H, L, device="cuda"), torch.rand(n_seq, H, L, device="cuda")
        if L >= 64:
            like = ("Gated DeltaNet scan", lambda: delta_rule_chunked_scan(q, k, v, g, beta))
        else:
            like = (None, None)
        tb.pair(f"minGRU over {n_seq} x {L} rows", lambda: min_gru_packed(y, state, b, BF), *like, nbytes=14.0 * T * W + 8.0 * n_seq * W, like_bytes=8.0 * T * W)


def blocks(tb: Table, E=4096, ff=14336, H=32, KV=8, D=128, W=4096, vocab=32000):
    from ..models.llama import gated_activation
    from ..ops.gemm import linear, linear_residual
    from ..ops.norm import rms_norm
    from ..ops.residual_stream import add_norm_stream, glu_of_rows, project
    from ..utils.activation import ActivationFunctionEnum as A

    n3 = (H + 2 * KV) * D
    wn, w2 = _randn(E), _randn(E)
    wq, bq, wo = _randn(n3, E, scale=0.02), _randn(n3), _randn(E, H * D, scale=0.02)
    wz, bz = _randn(3 * W, E, scale=0.02), _randn(3 * W)
    wl = _randn(H * (D + 64) + 576, E, scale=0.02)
    wgu, wd = _randn(2 * ff, E, scale=0.02), _randn(E, ff, scale=0.02)
    for T in (64, 8192):
        x, y, xb, h, a = _randn(T, E, dtype=F32), _randn(T, E, dtype=F32), _randn(T, E), _randn(T, E), _randn(T, ff)
        gu = _randn(T, 2 * ff)
        g = lambda n, k, out: dict(flops=2.0 * T * n * k, nbytes=2.0 * (T * k + n * k) + out)  # noqa: E731
        like = lambda n, k, out: dict(like_flops=2.0 * T * n * k, like_bytes=2.0 * (T * k + n * k) + out)  # noqa: E731
        tb.pair(f"T={T}: norm, add to the fp32 stream, norm", lambda: add_norm_stream(x, y, wn, w2, 1e-6), "Llama RMS norm", lambda: rms_norm(xb, wn),
                nbytes=14.0 * T * E, like_bytes=4.0 * T * E)
        tb.pair(f"T={T}: q, k, v with bias", lambda: project(h, wq, bias=bq), "Llama q, k, v in one product", lambda: linear(h, wq), **g(n3, E, 2.0 * T * n3),
                **like(n3, E, 2.0 * T * n3))
        n = wl.shape[0]
        tb.pair(f"T={T}: latent q and down projection", lambda: project(h, wl), "Llama q, k, v in one product", lambda: linear(h, wq), **g(n, E, 2.0 * T * n),
                **like(n3, E, 2.0 * T * n3))
        tb.pair(f"T={T}: minGRU z, x, g to fp32 with bias", lambda: project(h, wz, bias=bz, out_dtype=F32), "Llama q, k, v in one product", lambda: linear(h, wq),
                **g(3 * W, E, 12.0 * T * W), **like(n3, E, 2.0 * T * n3))
        tb.pair(f"T={T}: output projection to fp32", lambda: project(h, wo, out_dtype=F32), "Llama output projection + bf16 residual",
                lambda: linear_residual(h, wo, None, xb), **g(E, H * D, 4.0 * T * E), **like(E, H * D, 4.0 * T * E))
        tb.pair(f"T={T}: gate and up in one product", lambda: project(h, wgu), "Llama up projection", lambda: linear(h, wgu[:ff]), **g(2 * ff, E, 4.0 * T * ff),
                **like(ff, E, 2.0 * T * ff))
        tb.pair(f"T={T}: gelu gate", lambda: glu_of_rows(gu, ff, A.gelu_new), "Llama silu gate", lambda: gated_activation(gu[:, :ff], gu[:, ff:], A.silu),
                nbytes=6.0 * T * ff)
        tb.pair(f"T={T}: down projection to fp32", lambda: project(a, wd, out_dtype=F32), "Llama down projection + bf16 residual",
                lambda: linear_residual(a, wd, None, xb), **g(E, ff, 4.0 * T * E), **like(E, ff, 4.0 * T * E))


def kernel_table() -> dict:
    tb = Table()
    with torch.no_grad():
        for part in (attention, around_attention, recurrence, blocks):
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
