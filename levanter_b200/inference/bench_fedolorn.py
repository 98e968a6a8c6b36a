"""Fedolorn's serving kernels beside the like kernels of the closest models (Llama: attention, projections, norms; Mixtral: experts)
at equal sizes: ``python -m levanter_b200.inference.bench_fedolorn``, or ``bench.py --mode fedolorn``, which adds the engine's prefill
and decode throughput.

Every pair is timed with CUDA events, with a buffer larger than L2 rewritten before each timed call, and each kernel is set
against its own roofline: the larger of bytes that must move / measured HBM bandwidth and FLOPs / measured bf16 rate.
``distance`` is how many times further from its roofline the new kernel is than the like one."""
from __future__ import annotations

import argparse
import json
import statistics

import torch

from ..ops import lib
from ..ops.bench_kernels import _peaks

BF, F32 = torch.bfloat16, torch.float32


def _randn(*shape, dtype=BF, scale=1.0):
    return torch.randn(*shape, device="cuda", dtype=F32).mul_(scale).to(dtype)


class Timer:
    def __init__(self, iters: int = 15, warmup: int = 4):
        self.iters, self.warmup = iters, warmup
        self.flush = torch.empty(1 << 30, dtype=torch.uint8, device="cuda")  # its rewrite also covers the host time of the launch

    def __call__(self, fn) -> float:
        for _ in range(self.warmup):
            fn()
        times = []
        for _ in range(self.iters):
            self.flush.fill_(1)
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            fn()
            e1.record()
            torch.cuda.synchronize()
            times.append(e0.elapsed_time(e1))
        return statistics.median(times)


class Table:
    def __init__(self):
        self.timer, self.rows = Timer(), []
        self.tflops, self.gbs, self.how = _peaks()

    def _frac(self, ms, flops, nbytes):
        return max(flops / (self.tflops * 1e9), nbytes / (self.gbs * 1e6)) / ms

    def pair(self, name, new, like_name=None, like=None, *, flops=0.0, nbytes=0.0, like_flops=None, like_bytes=None):
        ms = self.timer(new)
        row = {"kernel": name, "us": round(ms * 1e3, 1), "roofline": round(self._frac(ms, flops, nbytes), 3)}
        if like is not None:
            m2 = self.timer(like)
            f2 = self._frac(m2, flops if like_flops is None else like_flops, nbytes if like_bytes is None else like_bytes)
            row.update({"like": like_name, "like_us": round(m2 * 1e3, 1), "like_roofline": round(f2, 3), "distance": round(f2 / self._frac(ms, flops, nbytes), 2)})
        self.rows.append(row)


def _pages(S, ctx, page, KV, width, dtype=BF):
    """Pages of S sequences of ctx tokens and the device tables of a decode round over them."""
    from .page_table import PageTable

    per = -(-ctx // page) + 1
    t = PageTable.init(S * per, S, page, per)
    slots, pos = [], []
    for s in range(S):
        t, _ = t.assign_seq_id_to_seq(s)
        slots += [s] * ctx
        pos += list(range(ctx))
    t, _ = t.allocate_for_seq(slots, pos)
    _, b = t.allocate_for_seq(list(range(S)), [ctx] * S)
    return _randn(S * per, page, KV, width, dtype=dtype), b.to("cuda")


def attention(tb: Table, T=8192, n_seq=4, H=32, KV=8, S=64, ctx=4096):
    from ..layers.attention import AttentionMask, dot_product_attention
    from ..ops import flash_attention as FA
    from ..ops import paged_attention as PA

    L = T // n_seq
    pos = (torch.arange(T, device="cuda") % L).int()
    seg = (torch.arange(T, device="cuda") // L).int()
    for dk, dv, chunk in ((128, 128, None), (128, 128, 1024), (128, 128, 256), (96, 96, None), (64, 64, None), (128, 64, 1024)):
        y = _randn(T, H * dk + KV * (dk + dv) + H * dv)
        q, k, v = (y[:, a:a + h * d].unflatten(1, (h, d)) for a, h, d in ((0, H, dk), (H * dk, KV, dk), ((H + KV) * dk, KV, dv)))
        gate = y[:, (H + KV) * dk + KV * dv:]
        c = chunk or L
        keys = n_seq * (L // c) * c * (c + 1) / 2
        flops = 2.0 * H * (dk + dv) * keys
        d = 64 if max(dk, dv) <= 64 else 128
        ql, kl, vl = (_randn(1, T, h, d) for h in (H, KV, KV))
        m = AttentionMask.causal().with_segment_ids(seg[None], sorted=True)
        tb.pair(f"prefill attention {dk}/{dv}, chunk {chunk or 'none'}, gated",
                lambda: FA.flash_attention_packed(q, k, v, pos, scaling_factor=dk ** -0.5, chunk=chunk, gate=gate), f"Llama prefill attention {d}",
                lambda: dot_product_attention(ql, kl, vl, m), flops=flops, nbytes=2.0 * (y.numel() + T * H * dv),
                like_flops=4.0 * H * d * n_seq * L * (L + 1) / 2, like_bytes=4.0 * T * (H + KV) * d)
    for dk, dv, chunk in ((128, 128, None), (128, 128, 1024), (96, 96, None), (64, 64, None), (192, 128, None)):
        kv, b = _pages(S, ctx - 1, 16, KV, dk + dv)
        q, gate = _randn(S, H, dk), _randn(S, H * dv)
        seen = ctx if chunk is None else (ctx - 1) % chunk + 1
        nb = 2.0 * S * (seen * KV * (dk + dv) + H * (dk + 2 * dv))
        d = 64 if max(dk, dv) <= 64 else 128
        kvl, bl = _pages(S, ctx - 1, 16, KV, 2 * d)
        kvl = kvl.view(kvl.shape[0], 16, 2 * KV, d)
        ql = _randn(S, H, d)
        tb.pair(f"decode attention {dk}/{dv}, chunk {chunk or 'none'}, {seen} keys, gated",
                lambda: PA.paged_attention_general(q, kv, KV, dv, b, sm_scale=dk ** -0.5, chunk=chunk, gate=gate), f"Llama decode attention {d}, {ctx} keys",
                lambda: PA.ragged_paged_attention(ql, kvl, bl.seq_lens, bl.page_indices, bl.cu_q_lens, bl.num_seqs, sm_scale=d ** -0.5),
                nbytes=nb, like_bytes=2.0 * S * (ctx * KV * 2 * d + 2 * H * d))
    kv, b = _pages(S, 64, 16, KV, 256)
    kvl = kv.view(kv.shape[0], 16, 2 * KV, 128)
    y = _randn(S, 2 * KV * 128)
    k, v = y[:, :KV * 128].unflatten(1, (KV, 128)), y[:, KV * 128:].unflatten(1, (KV, 128))
    k2, v2 = k.contiguous(), v.contiguous()
    tb.pair("cache write (strided rows)", lambda: PA.kv_page_write_general(kv, k, v, b.new_token_dests), "Llama cache write",
            lambda: PA.kv_page_write(kvl, k2, v2, b.new_token_dests), nbytes=4.0 * S * KV * 256)



def projections(tb: Table, E=4096, H=32, KV=8, D=128, ff=14336):
    from ..ops.embedding import embedding
    from ..ops.gemm import linear, linear_residual
    from ..ops.norm import rms_norm
    from ..ops.residual_stream import add_linear, embed_stream, project, rms_norm_stream

    table, wn = _randn(32000, E), _randn(E, scale=0.1)
    wq, wk, wv = _randn(H * D, E, scale=0.02), _randn(KV * D, E, scale=0.02), _randn(KV * D, E, scale=0.02)
    wf, wo = _randn((2 * H + 2 * KV) * D, E, scale=0.02), _randn(E, H * D, scale=0.02)
    up, down = _randn(ff, E, scale=0.02), _randn(E, ff, scale=0.02)
    for T in (64, 8192):
        x, xb, h, a = _randn(T, E, dtype=F32), _randn(T, E), _randn(T, E), _randn(T, ff)
        ids = torch.randint(0, 32000, (T,), device="cuda", dtype=torch.int32)
        g = lambda n, k, out: dict(flops=2.0 * T * n * k, nbytes=2.0 * (T * k + n * k) + out)  # noqa: E731
        like = lambda n, k, out: dict(like_flops=2.0 * T * n * k, like_bytes=2.0 * (T * k + n * k) + out)  # noqa: E731
        tb.pair(f"T={T}: embedding to the fp32 stream", lambda: embed_stream(ids, table, 8.0), "Llama embedding", lambda: embedding(ids, table),
                nbytes=6.0 * T * E, like_bytes=4.0 * T * E)
        tb.pair(f"T={T}: RMS norm of the fp32 stream", lambda: rms_norm_stream(x, wn, 1e-5, w_offset=1.0), "Llama RMS norm", lambda: rms_norm(xb, wn),
                nbytes=6.0 * T * E, like_bytes=4.0 * T * E)
        n, n3 = wf.shape[0], (H + 2 * KV) * D
        tb.pair(f"T={T}: q, k, v, gate in one product", lambda: project(h, wf), "Llama q, k, v products", lambda: (linear(h, wq), linear(h, wk), linear(h, wv)),
                **g(n, E, 2.0 * T * n), **like(n3, E, 2.0 * T * n3))
        tb.pair(f"T={T}: output projection + fp32 stream", lambda: add_linear(x, h, wo), "Llama output projection + bf16 residual",
                lambda: linear_residual(h, wo, None, xb), **g(E, H * D, 8.0 * T * E), **like(E, H * D, 4.0 * T * E))
        tb.pair(f"T={T}: up projection, squared relu", lambda: project(h, up, squared_relu=True), "Llama up projection", lambda: linear(h, up),
                **g(ff, E, 2.0 * T * ff), **like(ff, E, 2.0 * T * ff))
        tb.pair(f"T={T}: down projection + fp32 stream", lambda: add_linear(x, a, down), "Llama down projection + bf16 residual",
                lambda: linear_residual(a, down, None, xb), **g(E, ff, 8.0 * T * E), **like(E, ff, 4.0 * T * E))


def experts(tb: Table, E=4096, ff=1536, n=64, k=8, groups=8, keep=4):
    from ..ops import moe
    from ..ops.moe import RoutedTokens

    up, down = _randn(n, ff, E, scale=0.02), _randn(n, E, ff, scale=0.02)
    corr = _randn(n, scale=0.1)
    for T in (8, 64, 256, 8192):
        h, x = _randn(T, E), _randn(T, E, dtype=F32)
        z = _randn(T, n, dtype=F32)
        tb.pair(f"T={T}: sigmoid routing in groups, {n} experts", lambda: moe.route_sigmoid(z, corr, k, groups=groups, keep=keep), "Mixtral routing",
                lambda: moe.moe_route(z, k), nbytes=T * (4.0 * n + 8 * k), like_bytes=T * (8.0 * n + 8 * k))
        r = moe.route_sigmoid(z, corr, k, groups=groups, keep=keep)
        used = int((r.counts[:n] > 0).sum())
        # the two expert products on rows that are already in the padded layout, against Mixtral's grouped product of one matrix
        dest, offsets, tg, cap = moe.padded_layout(r.idx.reshape(-1), n)
        xp = h.new_zeros(cap, E).index_copy(0, dest, h.repeat_interleave(k, dim=0))
        fl, wb = 2.0 * T * k * ff * E, 2.0 * used * ff * E
        counts = r.counts.clone()

        def layer():
            counts[n:] = 0
            moe.add_expert_outputs(x, h, RoutedTokens(r.idx, r.w, counts), up, down)

        rows = moe._block_rows(T * k, n)
        bl = (T * k + min(n, T * k) * (rows - 1) + rows - 1) // rows
        tile = torch.full((bl,), -1, dtype=torch.int32, device="cuda")
        per = (r.counts[:n].long() + rows - 1) // rows
        tile[:int(per.sum())] = torch.repeat_interleave(torch.arange(n, device="cuda"), per).int()
        a = _randn(bl * rows, E)
        like = lambda: moe.grouped_linear(xp, up, tg, offsets)  # noqa: E731
        tb.pair(f"T={T}: expert up product, squared relu, {used} experts in blocks of {rows}", lambda: moe.grouped_product(a, up, tile, rows, True),
                "Mixtral grouped product", like, flops=fl, nbytes=wb + 2.0 * T * k * (E + ff))
        a2 = _randn(bl * rows, ff)
        xd = _randn(cap, ff)
        tb.pair(f"T={T}: expert down product", lambda: moe.grouped_product(a2, down, tile, rows, False), "Mixtral grouped product (down)",
                lambda: moe.grouped_linear(xd, down, tg, offsets), flops=fl, nbytes=wb + 2.0 * T * k * (E + ff))
        tb.pair(f"T={T}: whole expert layer after routing (dispatch, products, combine)", layer, flops=2 * fl, nbytes=2 * wb + 8.0 * T * E)


def kernel_table() -> dict:
    tb = Table()
    with torch.no_grad():
        for part in (attention, projections, experts):
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
