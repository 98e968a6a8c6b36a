"""Prefill and decode throughput of the inference engine on one GPU:
``python -m levanter_b200.inference.bench_decode --model llama3_8b --seqs 64 --prompt-len 512 --new-tokens 128 [--cuda-graph]``,
or tensor-parallel over the GPUs of one node (one rank per GPU, heads / KV heads / MLP columns split over the ranks):
``python -m torch.distributed.run --nproc-per-node 8 --master-addr 127.0.0.1 -m levanter_b200.inference.bench_decode --tp 8 --seqs 256
--prompt-min 128 --prompt-max 2048 --new-tokens 256 --cuda-graph``.

Random-init weights of the named architecture in bf16, synthetic uniform-random prompts, greedy decoding with stop tokens
disabled, so that every request produces exactly ``--new-tokens`` tokens.  The engine's own public entry point
(``InferenceEngine.generate``) is what is timed; phase times come from ``engine.stats`` (host clock after a device
synchronisation at the phase boundaries).  Prints one JSON line."""
from __future__ import annotations

import argparse
import json
import time

import numpy as np
import torch

MODELS = {
    "llama3_8b": dict(hidden_dim=4096, intermediate_dim=14336, num_layers=32, num_heads=32, num_kv_heads=8, vocab=128256),
    "llama2_7b": dict(hidden_dim=4096, intermediate_dim=11008, num_layers=32, num_heads=32, num_kv_heads=32, vocab=32000),
    "llama_1b": dict(hidden_dim=2048, intermediate_dim=8192, num_layers=16, num_heads=32, num_kv_heads=8, vocab=128256),
    # Fedolorn at the size of llama3_8b: the same width, heads, layers and vocabulary; with an attention gate and two feed-forward
    # matrices instead of a gated three, ff = 19456 gives a layer the same number of parameters.  The second one has 64 experts
    "fedolorn_8b": dict(family="fedolorn", hidden_dim=4096, num_layers=32, intermediate_dim=19456, vocab=128256),
    "fedolorn_moe": dict(family="fedolorn", hidden_dim=4096, num_layers=16, intermediate_dim=1536, vocab=128256,
                         moe=dict(num_experts=64, num_experts_per_tok=8, expert_groups=8, expert_groups_kept=4, router_scale=1.5)),
    "tiny_fedolorn": dict(family="fedolorn", hidden_dim=256, num_layers=2, intermediate_dim=64, vocab=1024,
                          heads=dict(num_heads=4, num_kv_heads=2, head_dim=64, v_head_dim=64, attention_scale=0.125, chunk_size=96),
                          moe=dict(num_experts=8, num_experts_per_tok=2, expert_groups=2, expert_groups_kept=1)),
    # Zadepel at the size of llama3_8b: the same width, layers, vocabulary, feed-forward and attention heads; a group of four layers is
    # attention, latent attention, minGRU, latent attention
    "zadepel_8b": dict(family="zadepel", hidden_dim=4096, num_layers=32, intermediate_dim=14336, vocab=128256),
    "tiny_zadepel": dict(family="zadepel", hidden_dim=256, num_layers=4, intermediate_dim=512, vocab=1024,
                         attention=dict(num_heads=4, num_kv_heads=2, head_dim=64, v_head_dim=64, attention_scale=0.125, rotary_dim=32), mingru=dict(width=320),
                         latent=dict(num_heads=4, head_dim=32, rotary_dim=16, v_head_dim=48, kv_lora_rank=64, attention_scale=0.15, sliding_window=96)),
    # Zosipel beside fedolorn_moe: the same width, vocabulary, layer runs and expert weights (three matrices of 1024 instead of two of 1536), a
    # shared expert, four of twelve layers run twice; of four layers one is differential attention in a window, three are latent attention
    "zosipel_moe": dict(family="zosipel", hidden_dim=4096, num_layers=12, intermediate_dim=1024, vocab=128256, shared=2048, loop=(4, 8, 2)),
    "tiny_zosipel": dict(family="zosipel", hidden_dim=256, num_layers=4, intermediate_dim=64, vocab=1024, shared=96, loop=(1, 3, 2),
                         attention=dict(num_heads=4, num_kv_heads=2, head_dim=32, v_head_dim=64, attention_scale=0.18, sliding_window=96, soft_cap=20.0),
                         latent=dict(num_heads=4, head_dim=48, v_head_dim=32, kv_lora_rank=64, attention_scale=0.15),
                         moe=dict(num_experts=8, num_experts_per_tok=2, expert_groups=4, expert_groups_kept=2)),
    # Mumizen at the size of zadepel_8b and, with mixtures, of zosipel_moe (as many layers as that has layer runs): a group of four layers is
    # lightning, latent attention, retention, latent attention that reads the latents of the other
    "mumizen_8b": dict(family="mumizen", hidden_dim=4096, num_layers=32, intermediate_dim=14336, vocab=128256),
    "mumizen_moe": dict(family="mumizen", hidden_dim=4096, num_layers=16, intermediate_dim=1024, vocab=128256,
                        moe=dict(num_experts=64, num_experts_per_tok=8, shared_intermediate_dim=2048)),
    "tiny_mumizen": dict(family="mumizen", hidden_dim=256, num_layers=6, intermediate_dim=64, vocab=1024, linear=(4, 64),
                         latent=dict(num_heads=4, head_dim=48, rotary_dim=16, v_head_dim=32, q_lora_rank=96, kv_lora_rank=64, attention_scale=0.125),
                         moe=dict(num_experts=8, num_experts_per_tok=2, shared_intermediate_dim=96)),
    "tiny": dict(hidden_dim=256, intermediate_dim=512, num_layers=2, num_heads=4, num_kv_heads=2, vocab=1024),
}


def model_config(m: dict, seq_len: int):
    """The model config of a ``MODELS`` entry (without its ``vocab``)."""
    m = dict(m)
    family = m.pop("family", "llama")
    if family == "llama":
        from ..models.llama import LlamaConfig

        return LlamaConfig(seq_len=seq_len, gradient_checkpointing=False, **m)
    if family == "zadepel":
        from ..models.zadepel import ZadepelConfig, ZadepelLayerConfig

        ff = m["intermediate_dim"]
        latent = dict(num_heads=32, head_dim=128, rotary_dim=64, v_head_dim=128, kv_lora_rank=512, attention_scale=192 ** -0.5, sliding_window=1024)
        latent = ZadepelLayerConfig(mixer="latent_attention", intermediate_dim=ff, **m.get("latent", latent))
        group = [ZadepelLayerConfig(mixer="attention", intermediate_dim=ff, **m.get("attention", {})), latent,
                 ZadepelLayerConfig(mixer="mingru", intermediate_dim=ff, **m.get("mingru", dict(width=4096))), latent]
        return ZadepelConfig(seq_len=seq_len, hidden_dim=m["hidden_dim"], gradient_checkpointing=False,
                             layers=tuple(group[i % 4] for i in range(m["num_layers"])))
    if family == "zosipel":
        from ..layers.rotary import PartialYarnRotaryEmbeddingsConfig
        from ..models.zosipel import ZosipelConfig, ZosipelLayerConfig

        moe = dict(intermediate_dim=m["intermediate_dim"], shared_intermediate_dim=m["shared"],
                   **m.get("moe", dict(num_experts=64, num_experts_per_tok=8, expert_groups=8, expert_groups_kept=4)))
        rope = PartialYarnRotaryEmbeddingsConfig(theta=500000.0, factor=4.0, original_max_position_embeddings=2048)
        attn = dict(num_heads=32, num_kv_heads=8, head_dim=64, v_head_dim=128, attention_scale=0.125, sliding_window=1024, soft_cap=30.0)
        latent = dict(num_heads=32, head_dim=128, v_head_dim=128, kv_lora_rank=512, attention_scale=128 ** -0.5)
        layers = {False: ZosipelLayerConfig(mixer="latent_attention", rope=None, **m.get("latent", latent), **moe),
                  True: ZosipelLayerConfig(mixer="attention", rope=rope, difference=0.5, **m.get("attention", attn), **moe)}
        start, stop, times = m["loop"] if m["num_layers"] >= m["loop"][1] else (0, 0, 0)
        return ZosipelConfig(seq_len=seq_len, hidden_dim=m["hidden_dim"], gradient_checkpointing=False, loop_start=start, loop_stop=stop, loop_times=times,
                             layers=tuple(layers[i % 4 == 2] for i in range(m["num_layers"])))
    if family == "mumizen":
        from ..layers.rotary import PartialYarnRotaryEmbeddingsConfig
        from ..models.mumizen import MumizenConfig, MumizenLayerConfig

        ff = dict(intermediate_dim=m["intermediate_dim"], **m.get("moe", {}))
        heads, d = m.get("linear", (32, 128))
        linear = dict(num_heads=heads, head_dim=d, v_head_dim=d, decay=tuple(1.0 - 2.0 ** (-3.0 - 5.0 * i / heads) for i in range(heads)), **ff)
        rope = PartialYarnRotaryEmbeddingsConfig(theta=500000.0, factor=4.0, original_max_position_embeddings=2048)
        latent = dict(mixer="latent_attention", rope=rope, **m.get("latent", dict(num_heads=32, head_dim=128, rotary_dim=64, v_head_dim=128, q_lora_rank=1536,
                                                                                  kv_lora_rank=512, attention_scale=192 ** -0.5)), **ff)
        group = [MumizenLayerConfig(mixer="lightning", **linear), MumizenLayerConfig(**latent), MumizenLayerConfig(mixer="retention", **linear), None]
        layers = [group[i % 4] or MumizenLayerConfig(kv_from=i - 2, **latent) for i in range(m["num_layers"])]
        return MumizenConfig(seq_len=seq_len, hidden_dim=m["hidden_dim"], norm_groups=8, gradient_checkpointing=False, layers=tuple(layers))
    from ..models.fedolorn import FedolornConfig, FedolornLayerConfig

    layer = FedolornLayerConfig(intermediate_dim=m["intermediate_dim"], **m.get("heads", {}), **m.get("moe", {}))
    return FedolornConfig(seq_len=seq_len, hidden_dim=m["hidden_dim"], embedding_scale=8.0, gradient_checkpointing=False,
                          layers=(layer,) * m["num_layers"])


def main(argv=None):
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", choices=sorted(MODELS), default="llama3_8b")
    ap.add_argument("--seqs", type=int, default=64)
    ap.add_argument("--prompt-len", type=int, default=512)
    ap.add_argument("--new-tokens", type=int, default=128)
    ap.add_argument("--page-size", type=int, default=16)
    ap.add_argument("--max-rounds", type=int, default=16)
    ap.add_argument("--cuda-graph", action="store_true")
    ap.add_argument("--layers", type=int, default=None, help="override the number of layers (short profiler captures)")
    ap.add_argument("--repeats", type=int, default=2, help="timed generate() calls after one warm-up call")
    ap.add_argument("--tp", type=int, default=1, help="tensor-parallel ranks (launch with torchrun, one rank per GPU)")
    ap.add_argument("--prompt-min", type=int, default=0, help="with --prompt-max: prompt lengths uniform in [min, max]")
    ap.add_argument("--prompt-max", type=int, default=0)
    ap.add_argument("--quiet", action="store_true", help="return the result without printing it")
    a = ap.parse_args(argv)
    return run(a)


def run(a):
    import os

    from ..data.passthrough_tokenizer import PassthroughTokenizer
    from .engine import InferenceEngine, InferenceEngineConfig, Request
    from .jit_scheduler import SeqDecodingParams

    m = dict(MODELS[a.model])
    vocab = m.pop("vocab")
    if a.layers is not None:
        m["num_layers"] = a.layers
    prompt_max = a.prompt_max or a.prompt_len
    prompt_min = a.prompt_min or prompt_max
    total_len = prompt_max + a.new_tokens
    cfg = model_config(m, max(total_len, 128))
    rank, local_rank = int(os.environ.get("RANK", "0")), int(os.environ.get("LOCAL_RANK", "0"))
    if torch.cuda.is_available():
        torch.cuda.set_device(local_rank)
    dev = torch.device("cuda", local_rank) if torch.cuda.is_available() else torch.device("cpu")
    dtype = torch.bfloat16 if dev.type == "cuda" else torch.float32
    tp = None
    if a.tp > 1:
        import torch.distributed as dist

        from ..parallel.mesh import DeviceMesh
        from ..parallel.tp import TensorParallel, shard_full_state_

        if not dist.is_initialized():
            dist.init_process_group("nccl" if dev.type == "cuda" else "gloo")
        assert dist.get_world_size() == a.tp, "launch one rank per tensor-parallel shard"
        tp = TensorParallel.from_mesh(DeviceMesh(1, 1, a.tp))
        # every rank builds the same unsharded random weights, keeps its shard and drops the rest
        full = cfg.build(vocab, seed=0, device=dev, dtype=dtype).eval()
        model = cfg.build(vocab, seed=1, device=dev, dtype=dtype, tp=tp).eval()
        shard_full_state_(model, {n: p.detach() for n, p in full.named_parameters()}, tp)
        del full
        if dev.type == "cuda":
            torch.cuda.empty_cache()
    else:
        model = cfg.build(vocab, seed=0, device=dev, dtype=dtype).eval()
    pages_per_seq = -(-total_len // a.page_size) + 1
    ecfg = InferenceEngineConfig(max_pages=a.seqs * pages_per_seq + 8, max_seqs=a.seqs, page_size=a.page_size, max_pages_per_seq=pages_per_seq,
                                 compute_dtype=dtype, max_seqs_in_prefill=min(a.seqs, 16), max_prefill_size=16 * prompt_max,
                                 max_rounds=a.max_rounds, use_cuda_graph=a.cuda_graph)
    engine = InferenceEngine.from_model_with_config(model, PassthroughTokenizer(vocab), ecfg)
    rng = np.random.default_rng(0)

    def requests():
        out = []
        for i in range(a.seqs):
            n = int(rng.integers(prompt_min, prompt_max + 1))
            out.append(Request(prompt_tokens=rng.integers(1, vocab - 1, n).tolist(), request_id=i,
                               decode_params=SeqDecodingParams(max_num_tokens=n + a.new_tokens, stop_tokens=None, temperature=0.0, key=i),
                               n_generations=1))
        return out

    with torch.no_grad():
        engine.generate(requests())  # warm-up (kernel attributes, graph capture, allocator)
        runs = []
        for _ in range(a.repeats):
            engine.reset()
            for k in engine.stats:
                engine.stats[k] = 0
            if dev.type == "cuda":
                torch.cuda.synchronize()
            t0 = time.perf_counter()
            res = engine.generate(requests())
            if dev.type == "cuda":
                torch.cuda.synchronize()
            wall = time.perf_counter() - t0
            st = dict(engine.stats)
            runs.append({"wall_s": wall, "generated": res.total_generated,
                         **st})
    device_round_ms = None
    if a.cuda_graph and engine._graph is not None:
        # the captured round alone, replayed back to back with no host work in between: pure device time per round
        # (the tables left in its static inputs are those of the last real round; token destinations are rewritten in place)
        g = engine._graph.graph
        for _ in range(3):
            g.replay()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        for _ in range(20):
            g.replay()
        e1.record()
        torch.cuda.synchronize()
        device_round_ms = e0.elapsed_time(e1) / 20
    if tp is not None:
        # a phase lasts as long as its slowest rank
        import torch.distributed as dist

        for r in runs:
            t = torch.tensor([r["wall_s"], r["prefill_seconds"], r["decode_seconds"]], dtype=torch.float64, device=dev)
            dist.all_reduce(t, op=dist.ReduceOp.MAX)
            r["wall_s"], r["prefill_seconds"], r["decode_seconds"] = (float(x) for x in t)
    best = min(runs, key=lambda r: r["wall_s"])
    out = {"metric": f"decode tokens/s (engine.generate, {a.tp} GPU{'s, tensor parallel' if a.tp > 1 else ''})", "model": a.model, "seqs": a.seqs,
           "prompt_len": a.prompt_len if not a.prompt_max else [prompt_min, prompt_max], "tp": a.tp,
           "kernel_all_reduces": None if tp is None else tp.kernel_all_reduces,
           "new_tokens": a.new_tokens, "page_size": a.page_size, "cuda_graph": bool(a.cuda_graph), "max_rounds": a.max_rounds, "dtype": str(dtype),
           "prefill_tokens_per_s": round(best["prefill_tokens"] / max(best["prefill_seconds"], 1e-9), 1),
           "decode_tokens_per_s": round(best["decode_tokens"] / max(best["decode_seconds"], 1e-9), 1),
           "end_to_end_generated_tokens_per_s": round(best["generated"] / best["wall_s"], 1),
           "ms_per_decode_round": round(1e3 * best["decode_seconds"] / max(best.get("decode_rounds", 0), 1), 3),
           "device_ms_per_round_graph_only": None if device_round_ms is None else round(device_round_ms, 3), "runs": runs}
    if rank == 0 and not a.quiet:
        print(json.dumps(out))
    return out


if __name__ == "__main__":
    main()
