"""Fedolorn through the framework (registry, checkpoint loading, engine, scheduler, trace replay) against ``fedolorn_oracle``: on
the CPU in fp32, and on a B200 in fp32 and bf16."""
import dataclasses
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import fedolorn_oracle as O
from levanter_b200.compat.hf_checkpoints import HFCheckpointConverter
from levanter_b200.inference.engine import InferenceEngine, InferenceEngineConfig, Request
from levanter_b200.inference.jit_scheduler import SeqDecodingParams
from levanter_b200.models.fedolorn import FedolornConfig, FedolornLayerConfig, FedolornLMHeadModel
from levanter_b200.models.lm_model import LmConfig, LmExample

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
PLACES = [pytest.param(("cpu", torch.float32), id="cpu-f32"), pytest.param(("cuda", torch.float32), id="gpu-f32", marks=pytest.mark.gpu),
          pytest.param(("cuda", torch.bfloat16), id="gpu-bf16", marks=pytest.mark.gpu)]


def _attn(heads, kv, dim, vdim, chunk, scale):
    return dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, mask={"size": chunk})


def _moe(ff, experts, top, count, keep, scale):
    return dict(kind="moe", expert={"ff": ff}, router=dict(experts=experts, top=top, groups={"count": count, "keep": keep}, scale=scale))


def _config(name):
    """Small models that differ in every size and constant, from each other and from layer to layer."""
    if name == "mixed":
        layers = [(_attn(4, 2, 24, 16, 20, 0.3), dict(kind="dense", ff=56)), (_attn(6, 1, 16, 40, 7, 0.41), _moe(24, 12, 3, 4, 2, 1.7)),
                  (_attn(2, 2, 40, 8, 64, 0.2), None), (_attn(4, 4, 8, 24, 33, 0.5), _moe(16, 5, 1, 1, 1, 0.8))]
        return dict(architecture="Fedolorn", vocab=83, width=72, embedding={"scale": 2.5}, norm={"eps": 0.01},
                    layers=[dict(type="attention", mixer=m, mlp=f) for m, f in layers])
    layers = [(_attn(3, 3, 18, 10, 16, 0.37), _moe(10, 6, 2, 3, 1, 2.2)), (_attn(2, 1, 6, 14, 1000, 0.6), dict(kind="dense", ff=22)),
              (_attn(2, 1, 6, 14, 1, 0.6), _moe(14, 8, 4, 2, 2, 0.5))]
    return dict(architecture="Fedolorn", vocab=45, width=50, embedding={"scale": 0.75}, norm={"eps": 1e-4},
                layers=[dict(type="attention", mixer=m, mlp=f) for m, f in layers])


@pytest.fixture(scope="module")
def checkpoint(tmp_path_factory):
    from safetensors.torch import save_file

    made = {}

    def make(name):
        if name not in made:
            cfg = _config(name)
            W = O.random_weights(cfg, seed=len(name))
            d = tmp_path_factory.mktemp(name)
            (d / "config.json").write_text(json.dumps(cfg))
            save_file(W, str(d / "model.safetensors"))
            made[name] = (cfg, W, str(d))
        return made[name]

    return make


def _load(path, place):
    return HFCheckpointConverter.from_hf(path).load_pretrained(ref=path, dtype=place[1], device=place[0], resize_vocab_to_match_tokenizer=False).eval()


def _engine(model, place, *, max_seqs=6, page_size=4, pages_per_seq=48, max_pages=None, **kw):
    return InferenceEngine.from_model_with_config(model, None, InferenceEngineConfig(
        max_seqs=max_seqs, page_size=page_size, max_pages_per_seq=pages_per_seq, max_pages=max_pages, compute_dtype=place[1], **kw))


def _tokens(n, vocab, seed=0):
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


def _close(got, want, place, what=""):
    """Row by row: every row in fp32; in bf16 a router's close call may send a few rows another way."""
    got, want = torch.as_tensor(got).double().cpu(), want.double()
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    if place[1] == torch.float32:
        assert float(err.max()) < 3e-5, (what, int(err.argmax()), float(err.max()))
    else:
        assert float(err.median()) < 0.02 and float((err > 0.06).double().mean()) <= 0.15, (what, err)


def test_registry_config_and_checkpoint_names(checkpoint, tmp_path):
    cfg, W, path = checkpoint("mixed")
    assert LmConfig.get_known_choices()["fedolorn"] is FedolornConfig
    conv = HFCheckpointConverter.from_hf(path)
    c = conv.config_from_hf_checkpoint(path)
    assert isinstance(c, FedolornConfig) and c.num_layers == 4 and c.layers[2].intermediate_dim is None and c.layers[1].expert_groups_kept == 2
    assert c.to_hf_config(83) == cfg
    m = _load(path, ("cpu", torch.bfloat16))
    assert isinstance(m, FedolornLMHeadModel) and m.vocab_size == 83
    assert sum(p.numel() for p in m.parameters()) == sum(t.numel() for t in W.values()) == c.total_trainable_params(83)
    assert c.flops_per_token(83) > 0
    conv.save_pretrained(m, str(tmp_path / "out"), save_tokenizer=False)
    from safetensors.torch import load_file

    back = load_file(str(tmp_path / "out" / "model.safetensors"))
    assert back.keys() == W.keys() and all(torch.equal(back[k], W[k]) for k in W)
    assert json.loads((tmp_path / "out" / "config.json").read_text())["layers"] == cfg["layers"]


def test_config_from_yaml_and_rejected_configs():
    from levanter_b200 import config as lev_config

    c = lev_config.decode(LmConfig, {"type": "fedolorn", "hidden_dim": 32, "layers": [
        {"num_heads": 2, "num_kv_heads": 1, "head_dim": 8, "v_head_dim": 8, "intermediate_dim": 16},
        {"num_heads": 4, "num_kv_heads": 2, "head_dim": 8, "v_head_dim": 16, "intermediate_dim": 8, "num_experts": 4, "num_experts_per_tok": 2}]})
    assert isinstance(c, FedolornConfig) and all(isinstance(l, FedolornLayerConfig) for l in c.layers) and c.layers[1].num_experts == 4
    m = c.build(11, seed=0)
    assert m(torch.arange(5)[None]).shape == (1, 5, 11)
    for bad in (dict(num_heads=3, num_kv_heads=2), dict(num_experts=6, num_experts_per_tok=1, expert_groups=4),
                dict(num_experts=6, num_experts_per_tok=3, expert_groups=3, expert_groups_kept=1), dict(chunk_size=0)):
        with pytest.raises(ValueError):
            FedolornLayerConfig(**bad)
    entry = _config("mixed")
    entry["layers"][0]["type"] = "other"
    with pytest.raises(ValueError):
        FedolornConfig.from_hf_config(entry)


@pytest.mark.parametrize("name", ["mixed", "odd"])
@pytest.mark.parametrize("place", PLACES)
def test_full_forward(checkpoint, name, place):
    cfg, W, path = checkpoint(name)
    toks = _tokens(131, cfg["vocab"])
    m = _load(path, place)
    with torch.no_grad():
        got = m(torch.tensor([toks, toks[::-1]], device=place[0]))
    _close(got[0], O.logits(cfg, W, toks), place)
    _close(got[1], O.logits(cfg, W, toks[::-1]), place)


def test_training_gradients_and_packed_segments(checkpoint):
    """The differentiable path: gradients against finite differences of the oracle, and packed sequences restart their chunks."""
    cfg, W, path = checkpoint("mixed")
    m = _load(path, ("cpu", torch.float32))
    a, b = _tokens(30, 83, 1), _tokens(45, 83, 2)
    seg = torch.tensor([0] * 30 + [1] * 45)
    ex = LmExample.causal(torch.tensor(a + b), segment_ids=seg)
    with torch.no_grad():
        got = m(ex.tokens[None], dataclasses.replace(ex.attn_mask, segment_ids=(seg[None], seg[None])))[0]
    _close(got, torch.cat([O.logits(cfg, W, a), O.logits(cfg, W, b)]), ("cpu", torch.float32))
    toks = torch.tensor(a)
    m.train()
    ref = torch.randn(30, 83, generator=torch.Generator().manual_seed(0), dtype=torch.float64)
    (m(toks[None])[0].double() * ref).sum().backward()
    params = dict(m.named_parameters())
    for pname in ("transformer.layers.0.self_attn.g_proj.weight", "transformer.layers.1.mlp.experts.up", "transformer.layers.1.mlp.router.weight",
                  "transformer.layers.3.post_attention_layernorm.weight", "embeddings.token_embeddings.weight"):
        d = torch.randn(params[pname].shape, generator=torch.Generator().manual_seed(1), dtype=torch.float64)
        names = m.hf_tensor_names(pname)
        vals = []
        for sgn in (1, -1):
            W2 = {k: v.double() for k, v in W.items()}
            for j, n in enumerate([names] if isinstance(names, str) else names):
                W2[n] = W2[n] + sgn * 1e-5 * (d if isinstance(names, str) else d[j])
            vals.append((O.logits(cfg, W2, a) * ref).sum())
        fd = float((vals[0] - vals[1]) / 2e-5)
        got = float((params[pname].grad.double() * d).sum())
        assert abs(got - fd) <= 2e-3 * max(abs(fd), 1.0), (pname, got, fd)


# ------------------------------------------------------------------------------------------------ serving
def _feed(eng, schedule):
    """Run ``schedule`` (a list of steps, each a list of ``(name, tokens)``) on caller-fed sequences; all logits per name."""
    slots, out = {}, {}
    for step in schedule:
        chunks = []
        for name, toks in step:
            if name not in slots:
                slots[name] = eng.open_sequence()
            chunks.append((slots[name], toks))
        n = sum(len(t) for _, t in step)
        logits = eng.forward_packed(chunks, list(range(n)))
        at = 0
        for name, toks in step:
            out.setdefault(name, []).append(logits[at:at + len(toks)].float().cpu())
            at += len(toks)
    return {k: torch.cat(v) for k, v in out.items()}, slots


def _cuts(toks, sizes):
    out, at, i = [], 0, 0
    while at < len(toks):
        n = sizes[i % len(sizes)]
        out.append(toks[at:at + n])
        at, i = at + n, i + 1
    return out


@pytest.mark.parametrize("name", ["mixed", "odd"])
@pytest.mark.parametrize("place", PLACES)
def test_prompt_portions_and_token_by_token(checkpoint, name, place):
    """The same sequence in one step, in portions of several sizes, and decoded one token at a time, across page and chunk borders
    of every layer; each form on pages that the previous one gave back."""
    cfg, W, path = checkpoint(name)
    m = _load(path, place)
    eng = _engine(m, place)
    toks = _tokens(137, cfg["vocab"], 5)
    want = O.logits(cfg, W, toks)
    for sizes in ([137], [64, 73], [2], [3, 1, 10], [20, 7], [33, 1], [1]):
        got, slots = _feed(eng, [[("a", c)] for c in _cuts(toks, sizes)])
        _close(got["a"], want, place, sizes)
        eng.close_sequences(slots.values())
    assert eng._free_page_count() == eng.config.imputed_max_pages and len(eng.free_slots) == eng.config.max_seqs


@pytest.mark.parametrize("place", PLACES)
def test_batches_against_each_alone(checkpoint, place):
    """Unequal requests in one batch, decoded together, with prompts starting while others decode and others ending; the pool is so
    small that every page is used several times."""
    cfg, W, path = checkpoint("mixed")
    m = _load(path, place)
    eng = _engine(m, place, max_seqs=4, max_pages=60)
    lens = {"a": 1, "b": 66, "c": 19, "d": 41}
    full = {k: _tokens(n + 25, cfg["vocab"], i) for i, (k, n) in enumerate(lens.items())}
    want = {k: O.logits(cfg, W, t) for k, t in full.items()}
    for _ in range(2):
        got, slots = _feed(eng, [[(k, full[k][:n]) for k, n in lens.items()]] +
                           [[(k, full[k][n + i:n + i + 1]) for k, n in lens.items()] for i in range(25)])
        for k in lens:
            _close(got[k], want[k], place, k)
        eng.close_sequences(slots.values())
    # ragged: one decodes, one goes on with a portion, one starts
    s = {k: eng.open_sequence() for k in "abc"}
    eng.forward_packed([(s["a"], full["a"][:5]), (s["b"], full["b"][:30])], [])
    rows = eng.forward_packed([(s["a"], full["a"][5:6]), (s["b"], full["b"][30:43]), (s["c"], full["c"][:22])], list(range(36))).float().cpu()
    for part, k, lo, hi in ((rows[:1], "a", 5, 6), (rows[1:14], "b", 30, 43), (rows[14:], "c", 0, 22)):
        _close(part, want[k][lo:hi], place, k)


@pytest.mark.parametrize("place", PLACES)
def test_greedy_generation_through_the_scheduler(checkpoint, place):
    """More requests than slots, clones, early stops, long decoding over several chunks of every layer."""
    cfg, W, path = checkpoint("mixed")
    m = _load(path, place)
    eng = _engine(m, place, max_seqs=3, pages_per_seq=40, max_pages=110, max_rounds=5, use_cuda_graph=place[0] == "cuda")
    prompts = [_tokens(n, cfg["vocab"], 10 + n) for n in (1, 19, 40, 7, 63)]
    new = 75
    reqs = [Request(p, i, SeqDecodingParams(len(p) + new, None, 0.0, i), 2 if i == 1 else 1) for i, p in enumerate(prompts)]
    for _ in range(2):  # the second run reuses slots and pages (and the captured graph)
        res = eng.generate(reqs)
        outs = {0: res.tokens[0:1], 1: res.tokens[1:3], 2: res.tokens[3:4], 3: res.tokens[4:5], 4: res.tokens[5:6]}
        for i, p in enumerate(prompts):
            for out in outs[i]:
                assert len(out) == new
                lg = O.logits(cfg, W, p + out[:-1])[len(p) - 1:]
                chosen = lg.gather(1, torch.tensor(out)[:, None]).squeeze(1)
                gap = (lg.max(dim=1).values - chosen) / lg.std(dim=1)  # 0 where the generated token is the arg-max
                if place[1] == torch.float32:
                    assert float(gap.max()) < 1e-4, (i, gap)
                else:
                    assert float((gap > 0.15).double().mean()) < 0.1, (i, gap)
    assert eng._free_page_count() == 110


@pytest.mark.parametrize("place", PLACES)
def test_trace_replay(checkpoint, place, tmp_path):
    """The command line: batches of requests, wanted places, requests that end, a later batch with more requests."""
    cfg, W, path = checkpoint("odd")
    full = {k: _tokens(n, cfg["vocab"], n) for k, n in (("p", 40), ("q", 23), ("r", 9), ("s", 30))}
    steps = [dict(step=0, entries=[dict(id="p", tokens=full["p"][:38], want=[0, 15, 16, 37])], end=[]),
             dict(step=1, entries=[dict(id="p", tokens=full["p"][38:39], want=[])], end=[]),
             dict(step=2, entries=[dict(id="p", tokens=full["p"][39:], want=[0])], end=["p"]),
             dict(step=3, entries=[dict(id=k, tokens=full[k][:-1], want=[len(full[k]) - 2]) for k in "qrs"], end=[]),
             dict(step=4, entries=[dict(id=k, tokens=full[k][-1:], want=[0]) for k in "srq"], end=["q", "r", "s"])]
    wanted = {0: [("p", 0), ("p", 15), ("p", 16), ("p", 37)], 2: [("p", 39)], 3: [("q", 21), ("r", 7), ("s", 28)], 4: [("s", 29), ("r", 8), ("q", 22)]}
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", str(place[1]).split(".")[1], "--out", str(tmp_path),
                        "--max-tokens", "70", "--device", place[0]], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True,
                       timeout=600, env={**os.environ, "PATH": os.path.dirname(sys.executable) + os.pathsep + os.environ["PATH"]})
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(5)]
    assert sorted(f for f in os.listdir(tmp_path) if f.endswith(".f32")) == ["0.f32", "2.f32", "3.f32", "4.f32"]
    want = {k: O.logits(cfg, W, t) for k, t in full.items()}
    for s, rows in wanted.items():
        got = torch.from_numpy(np.fromfile(tmp_path / f"{s}.f32", dtype="<f4").reshape(len(rows), cfg["vocab"]))
        _close(got, torch.stack([want[k][p] for k, p in rows]), place, s)


def test_chunk_masks():
    """The structured mask against the oracle's visibility: whole, by blocks, restarting in every packed segment."""
    from levanter_b200.layers.attention import AttentionMask, chunk_segments

    for n, chunk in ((40, 7), (33, 16), (20, 1), (12, 100)):
        see = AttentionMask.causal().with_chunk_size(chunk).materialize(n, n)
        assert torch.equal(see, O.visible(n, chunk))
        block = AttentionMask.causal().with_chunk_size(chunk).materialize(n, n, (5, 6), (3, 8))
        assert torch.equal(block, O.visible(n, chunk)[5:11, 3:11])
    seg = torch.tensor([[0] * 9 + [1] * 10 + [-1] * 3])
    assert chunk_segments(seg, 4).tolist() == [[0] * 4 + [1] * 4 + [2] + [3] * 4 + [4] * 4 + [5] * 2 + [-1] * 3]
    m = AttentionMask.causal().with_segment_ids(seg).with_chunk_size(4).materialize(22, 22)[0, 0]
    assert torch.equal(m[:9, :9], O.visible(9, 4)) and torch.equal(m[9:19, 9:19], O.visible(10, 4)) and not m[9:19, :9].any()
    with pytest.raises(ValueError):
        AttentionMask.causal().with_chunk_size(4) & AttentionMask.causal().with_chunk_size(5)


def test_sample_lm_command(checkpoint, tmp_path, monkeypatch, capsys):
    """The sampling command line on a checkpoint directory: greedy tokens are the oracle's."""
    from levanter_b200 import config as lev_config
    from levanter_b200.data.passthrough_tokenizer import PassthroughTokenizer
    from levanter_b200.main import sample_lm

    cfg, W, path = checkpoint("odd")
    monkeypatch.setattr(sample_lm, "load_tokenizer", lambda name: PassthroughTokenizer(cfg["vocab"]))
    monkeypatch.setattr(sample_lm, "local_device", lambda: torch.device("cpu"))
    prompt = _tokens(21, cfg["vocab"], 3)
    sample_lm.main(lev_config.decode(sample_lm.SampleLmConfig, {
        "hf_checkpoint": path, "tokenizer": "ids", "model": {"type": "fedolorn"}, "prompts": [" ".join(map(str, prompt))], "max_new_tokens": 12,
        "n_rounds": 1, "stop_sequence": None, "temperature": 0.0, "engine": {"max_seqs": 2, "page_size": 8, "max_pages_per_seq": 6, "compute_dtype": "float32"},
        "trainer": {"require_accelerator": False, "tracker": {"type": "noop"}, "log_dir": str(tmp_path), "mp": "f32"}}))
    out = capsys.readouterr().out
    toks = list(prompt)
    for _ in range(12):
        toks.append(int(O.logits(cfg, W, toks)[-1].argmax()))
    want = [t for t in toks[21:] if t != cfg["vocab"] - 1]  # the command drops the padding token
    got = out.split("Generated text for 0", 1)[1].split(":", 1)[1].split("\n")[0].split()
    assert [int(t) for t in got] == want
