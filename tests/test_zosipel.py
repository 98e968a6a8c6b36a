"""Zosipel through the framework (registry, checkpoint loading, engine, scheduler, trace replay) against ``zosipel_oracle``: on the CPU
in fp32, and on a B200 in fp32 and bf16."""
import dataclasses
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import zosipel_oracle as O
from levanter_b200.compat.hf_checkpoints import HFCheckpointConverter
from levanter_b200.inference.engine import Request
from levanter_b200.inference.jit_scheduler import SeqDecodingParams
from levanter_b200.layers.rotary import DefaultRotaryEmbeddingsConfig, PartialYarnRotaryEmbeddingsConfig
from levanter_b200.models.lm_model import LmConfig, LmExample
from levanter_b200.models.zosipel import ZosipelConfig, ZosipelLayerConfig, ZosipelLMHeadModel
from test_fedolorn import PLACES, ROOT, _cuts, _engine, _feed, _load, _tokens


def _attn(heads, kv, dim, vdim, scale, diff, dims, base, window=None, cap=None, yarn=None):
    m = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, diff=diff, rot=dict(base=base, dims=dims))
    if yarn is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    if window is not None:
        m["mask"] = {"size": window}
    if cap is not None:
        m["softcap"] = cap
    return dict(type="attention", mixer=m)


def _latent(heads, dim, vdim, rank, scale):
    return dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, vdim=vdim, kv_rank=rank, scale=scale))


def _moe(ff, experts, top, count, keep, shared=None):
    f = dict(kind="moe", expert={"ff": ff}, router=dict(experts=experts, top=top, groups={"count": count, "keep": keep}))
    return f if shared is None else dict(f, shared={"ff": shared})


def _config(name):
    """Small models that differ in every size and constant, from each other and from layer to layer."""
    if name == "mixed":  # layers before, within and after the loop; the loop begins with attention
        layers = [(_latent(5, 24, 32, 40, 0.25), _moe(24, 10, 3, 5, 2, 40)),
                  (_attn(4, 2, 16, 24, 0.3, 0.35, 8, 300.0, 20, 6.0, (8.0, 24, 4.0, 0.5)), _moe(16, 6, 2, 2, 1, 56)),
                  (_attn(6, 3, 24, 40, 0.25, 0.6, 24, 5000.0, 7, None, (3.0, 60, 16.0, 1.0)), None),
                  (_latent(3, 40, 16, 72, 0.2), _moe(32, 8, 2, 4, 4)),
                  (_attn(8, 1, 8, 16, 0.4, 0.2, 6, 50.0, None, 3.0), _moe(8, 9, 4, 3, 2, 24))]
        return _whole("Zosipel", 83, 72, 0.01, layers, dict(start=1, stop=4, times=3))
    if name == "odd":  # sizes that are not multiples of 8; a window wider than any sequence; the loop is the whole model
        layers = [(_attn(4, 2, 10, 18, 0.37, 0.45, 6, 40.0, 1000, 9.0, (2.0, 100, 8.0, 2.0)), _moe(10, 6, 2, 3, 2, 22)),
                  (_latent(3, 14, 10, 18, 0.3), _moe(14, 7, 3, 1, 1, 6)),
                  (_attn(3, 3, 6, 10, 0.5, 0.7, 2, 90.0, 33), None)]
        return _whole("Zosipel", 45, 50, 1e-4, layers, dict(start=0, stop=3, times=2))
    if name == "flat":  # no loop; many query heads per key/value head (more rows than a tensor-core tile)
        layers = [(_attn(18, 2, 16, 32, 0.25, 0.5, 16, 700.0, 45, 4.0), _moe(16, 4, 2, 2, 2, 16)), (_latent(18, 16, 32, 24, 0.3), None)]
        return _whole("Zosipel", 61, 64, 1e-5, layers, None)
    # one of everything: a window of one token, one head, one expert, one pass
    layers = [(_latent(1, 8, 8, 8, 1.0), None), (_attn(1, 1, 8, 8, 1.0, 0.1, 2, 10.0, 1, 1.0, (1.0, 16, 2.0, 1.0)), _moe(8, 1, 1, 1, 1, 8))]
    return _whole("Zosipel", 24, 16, 1e-6, layers, dict(start=1, stop=2, times=1))


def _whole(arch, vocab, width, eps, layers, loop):
    cfg = dict(architecture=arch, vocab=vocab, width=width, norm={"eps": eps}, layers=[dict(l, mlp=f) for l, f in layers])
    return cfg if loop is None else dict(cfg, loop=loop)


NAMES = ["mixed", "odd", "flat", "ones"]


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


def _close(got, want, place, what=""):
    """Row by row: every row in fp32; in bf16 a router's close call may send a few rows another way."""
    got, want = torch.as_tensor(got).double().cpu(), want.double()
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    if place[1] == torch.float32:
        assert float(err.max()) < 1e-4, (what, int(err.argmax()), float(err.max()))
    else:
        assert float(err.median()) < 0.05 and float((err > 0.15).double().mean()) <= 0.15, (what, int(err.argmax()), err)


def test_registry_config_and_checkpoint_names(checkpoint, tmp_path):
    cfg, W, path = checkpoint("mixed")
    assert LmConfig.get_known_choices()["zosipel"] is ZosipelConfig
    conv = HFCheckpointConverter.from_hf(path)
    c = conv.config_from_hf_checkpoint(path)
    assert isinstance(c, ZosipelConfig) and c.num_layers == 5 and c.layers[2].intermediate_dim is None and c.layers[2].sliding_window == 7
    assert isinstance(c.layers[1].rope, PartialYarnRotaryEmbeddingsConfig) and isinstance(c.layers[4].rope, DefaultRotaryEmbeddingsConfig)
    assert c.to_hf_config(83) == cfg
    assert [i for i, _ in c.layer_runs()] == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4] and [t for _, t in c.layer_runs() if t is not None] == [0, 1, 2]
    m = _load(path, ("cpu", torch.bfloat16))
    assert isinstance(m, ZosipelLMHeadModel) and m.vocab_size == 83
    assert sum(p.numel() for p in m.parameters()) == sum(t.numel() for t in W.values()) == c.total_trainable_params(83)
    assert c.flops_per_token(83) > 0
    assert len(m.initial_cache(4, 8)) == 11  # a cache for every run of a layer
    conv.save_pretrained(m, str(tmp_path / "out"), save_tokenizer=False)
    from safetensors.torch import load_file

    back = load_file(str(tmp_path / "out" / "model.safetensors"))
    assert back.keys() == W.keys() and all(torch.equal(back[k], W[k]) for k in W)
    assert json.loads((tmp_path / "out" / "config.json").read_text())["layers"] == cfg["layers"]
    flat = ZosipelConfig.from_hf_config(_config("flat"))
    assert flat.loop_times == 0 and flat.to_hf_config(61) == _config("flat")


def test_config_from_yaml_and_rejected_configs():
    from levanter_b200 import config as lev_config

    c = lev_config.decode(LmConfig, {"type": "zosipel", "hidden_dim": 32, "loop_start": 0, "loop_stop": 1, "loop_times": 2, "layers": [
        {"mixer": "attention", "num_heads": 2, "num_kv_heads": 1, "head_dim": 8, "v_head_dim": 8, "intermediate_dim": 16, "num_experts": 4,
         "num_experts_per_tok": 2, "rope": {"type": "yarn_partial", "theta": 100.0, "factor": 2.0, "rotary_dim": 4}},
        {"mixer": "latent_attention", "num_heads": 2, "head_dim": 8, "v_head_dim": 8, "kv_lora_rank": 8, "intermediate_dim": None}]})
    assert isinstance(c, ZosipelConfig) and all(isinstance(l, ZosipelLayerConfig) for l in c.layers) and c.layers[0].rope.factor == 2.0
    m = c.build(11, seed=0)
    assert m(torch.arange(5)[None]).shape == (1, 5, 11)
    for bad in (dict(num_heads=3, num_kv_heads=2), dict(mixer="other"), dict(rope=DefaultRotaryEmbeddingsConfig(rotary_dim=200)), dict(sliding_window=0),
                dict(rope=PartialYarnRotaryEmbeddingsConfig(rotary_dim=7)), dict(soft_cap=0.0), dict(num_experts=6, expert_groups=4),
                dict(num_experts=8, expert_groups=4, expert_groups_kept=1, num_experts_per_tok=3)):
        with pytest.raises(ValueError):
            ZosipelLayerConfig(**bad)
    for bad in (dict(loop_start=0, loop_stop=2, loop_times=1), dict(loop_start=1, loop_stop=1, loop_times=1), dict(layers=())):
        with pytest.raises(ValueError):
            ZosipelConfig(**bad)
    for change in (lambda l: l.update(type="other"), lambda l: l["mlp"].update(kind="other")):
        entry = _config("mixed")
        change(entry["layers"][1])
        with pytest.raises(ValueError):
            ZosipelConfig.from_hf_config(entry)


@pytest.mark.parametrize("dims,base,yarn", [(8, 300.0, (8.0, 24, 4.0, 0.5)), (64, 500000.0, (4.0, 2048, 32.0, 1.0)), (24, 5000.0, (3.0, 60, 16.0, 1.0)),
                                            (6, 40.0, (2.0, 100, 1e-3, 1e-4)), (16, 10.0, (1.0, 16, 2.0, 1.0)), (2, 90.0, (32.0, 7, 8.0, 8.0)), (10, 90.0, None)])
def test_rotation(dims, base, yarn):
    """Frequencies, ramp and magnitude, with ramps that are clipped at either end or empty, and the dimensions that pass."""
    rot = dict(base=base, dims=dims)
    c = DefaultRotaryEmbeddingsConfig(theta=base, rotary_dim=dims)
    if yarn is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
        c = PartialYarnRotaryEmbeddingsConfig(theta=base, rotary_dim=dims, factor=yarn[0], original_max_position_embeddings=yarn[1], beta_fast=yarn[2],
                                              beta_slow=yarn[3])
    r = c.build(dims + 6)
    f, mag = O.yarn(base, dims, rot.get("scaling"))
    assert torch.allclose(r.inv_freq.double(), torch.tensor(f, dtype=torch.float64), rtol=1e-6) and abs(r.temperature - mag) < 1e-12 and r.rotary_dim == dims
    x = torch.randn(40, 3, dims + 6, generator=torch.Generator().manual_seed(0), dtype=torch.float64)
    assert torch.allclose(r(x.float(), torch.arange(40) + 9).double(), O.rotate(x, rot, 9), atol=1e-4)


@pytest.mark.parametrize("name", NAMES)
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
    """The differentiable path: gradients against finite differences of the oracle (with and without recomputation), and packed
    sequences restart their windows."""
    cfg, W, path = checkpoint("mixed")
    m = _load(path, ("cpu", torch.float32))
    a, b = _tokens(30, 83, 1), _tokens(45, 83, 2)
    seg = torch.tensor([0] * 30 + [1] * 45)
    ex = LmExample.causal(torch.tensor(a + b), segment_ids=seg)
    with torch.no_grad():
        pos = torch.cat([torch.arange(30), torch.arange(45)])
        got = m(ex.tokens[None], dataclasses.replace(ex.attn_mask, segment_ids=(seg[None], seg[None])), pos_ids=pos)[0]
    _close(got, torch.cat([O.logits(cfg, W, a), O.logits(cfg, W, b)]), ("cpu", torch.float32))
    toks = torch.tensor(a)
    ref = torch.randn(30, 83, generator=torch.Generator().manual_seed(0), dtype=torch.float64)
    (m(toks[None])[0].double() * ref).sum().backward()
    kept = {n: p.grad.clone() for n, p in m.named_parameters()}
    m.zero_grad()
    m.train()
    (m(toks[None])[0].double() * ref).sum().backward()
    params = dict(m.named_parameters())
    assert all(torch.allclose(params[n].grad, g, rtol=1e-4, atol=1e-4 * float(g.abs().max())) for n, g in kept.items())
    for pname in ("transformer.loop_step", "transformer.layers.0.mixer.sinks", "transformer.layers.0.mixer.kv_b_proj.weight",
                  "transformer.layers.1.mixer.lambda_q1", "transformer.layers.2.mixer.lambda_k2", "transformer.layers.1.mixer.g_proj.weight",
                  "transformer.layers.2.mixer.k_proj.bias", "transformer.layers.1.mlp.experts.gate_up", "transformer.layers.1.mlp.router.weight",
                  "transformer.layers.4.mlp.shared_gate.weight", "transformer.layers.1.post_attention_layernorm.weight", "lm_head.weight"):
        d = torch.randn(params[pname].shape, generator=torch.Generator().manual_seed(1), dtype=torch.float64)
        vals = []
        for sgn in (1, -1):
            W2 = {k: v.double() for k, v in W.items()}
            for n, view, shape in m.hf_tensor_parts(pname, d):
                W2[n] = W2[n] + sgn * 1e-6 * view.reshape(shape)
            vals.append((O.logits(cfg, W2, a) * ref).sum())
        fd = float((vals[0] - vals[1]) / 2e-6)
        got = float((params[pname].grad.double() * d).sum())
        assert abs(got - fd) <= 2e-3 * max(abs(fd), 1.0), (pname, got, fd)


# ------------------------------------------------------------------------------------------------ serving
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("place", PLACES)
def test_prompt_portions_and_token_by_token(checkpoint, name, place):
    """The same sequence in one step, in portions of several sizes, and decoded one token at a time, across page and window borders
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
    for order in ("abcd", "dbca"):
        got, slots = _feed(eng, [[(k, full[k][:lens[k]]) for k in order]] + [[(k, full[k][lens[k] + i:lens[k] + i + 1]) for k in order] for i in range(25)])
        for k in lens:
            _close(got[k], want[k], place, k)
        eng.close_sequences(slots.values())
    # ragged: one decodes, one goes on with a portion, one starts
    s = {k: eng.open_sequence() for k in "abc"}
    eng.forward_packed([(s["a"], full["a"][:5]), (s["b"], full["b"][:30])], [])
    rows = eng.forward_packed([(s["a"], full["a"][5:6]), (s["b"], full["b"][30:43]), (s["c"], full["c"][:22])], list(range(36))).float().cpu()
    _close(rows, torch.cat([want["a"][5:6], want["b"][30:43], want["c"][:22]]), place, "ragged")
    # a request ends, its slot goes to a new one, the others go on
    eng.close_sequences([s["a"]])
    s["d"] = eng.open_sequence()
    assert s["d"] == s["a"]
    rows = eng.forward_packed([(s["d"], full["d"][:12]), (s["b"], full["b"][43:44])], list(range(13))).float().cpu()
    _close(rows, torch.cat([want["d"][:12], want["b"][43:44]]), place, "slot taken again")


@pytest.mark.parametrize("place", PLACES)
def test_greedy_generation_through_the_scheduler(checkpoint, place):
    """More requests than slots, clones, early stops, long decoding over several windows."""
    cfg, W, path = checkpoint("mixed")
    m = _load(path, place)
    eng = _engine(m, place, max_seqs=3, pages_per_seq=40, max_pages=110, max_rounds=5, use_cuda_graph=place[0] == "cuda")
    prompts = [_tokens(n, cfg["vocab"], 10 + n) for n in (1, 19, 40, 7, 63)]
    new = 75
    reqs = [Request(p, i, SeqDecodingParams(len(p) + new, None, 0.0, i), 2 if i == 1 else 1) for i, p in enumerate(prompts)]
    seen = {}
    for _ in range(2):  # the second run reuses slots and pages (and the captured graph)
        res = eng.generate(reqs)
        outs = {0: res.tokens[0:1], 1: res.tokens[1:3], 2: res.tokens[3:4], 3: res.tokens[4:5], 4: res.tokens[5:6]}
        for i, p in enumerate(prompts):
            for out in outs[i]:
                assert len(out) == new
                if (i, tuple(out)) in seen:
                    continue
                lg = seen[i, tuple(out)] = O.logits(cfg, W, p + out[:-1])[len(p) - 1:]
                chosen = lg.gather(1, torch.tensor(out)[:, None]).squeeze(1)
                gap = (lg.max(dim=1).values - chosen) / lg.std(dim=1)  # 0 where the generated token is the arg-max
                # over some hundred tokens a router's close call may go the other way even in fp32
                if place[1] == torch.float32:
                    assert float((gap > 1e-3).double().mean()) < 0.05, (i, gap)
                else:
                    assert float((gap > 0.3).double().mean()) < 0.1, (i, gap)
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
    want = {k: O.logits(cfg, W, t) for k, t in full.items()}
    got, ref = [], []
    for s, rows in wanted.items():
        got.append(torch.from_numpy(np.fromfile(tmp_path / f"{s}.f32", dtype="<f4").reshape(len(rows), cfg["vocab"])))
        ref.append(torch.stack([want[k][p] for k, p in rows]))
    _close(torch.cat(got), torch.cat(ref), place)


@pytest.mark.parametrize("place", PLACES)
def test_weights_that_change_after_serving(checkpoint, place):
    """Derived weights (joint projections, whole-key products, the second map's weight, sinks) follow their parameters: the same engine
    after a load of other weights."""
    cfg, W, path = checkpoint("mixed")
    m = _load(path, place)
    eng = _engine(m, place)
    toks = _tokens(24, cfg["vocab"], 8)
    got, slots = _feed(eng, [[("a", toks)]])
    _close(got["a"], O.logits(cfg, W, toks), place)
    eng.close_sequences(slots.values())
    other = O.random_weights(cfg, seed=77)
    from levanter_b200.compat.hf_checkpoints import load_hf_state_dict

    load_hf_state_dict(m, other)
    got, _ = _feed(eng, [[("a", toks)]])
    _close(got["a"], O.logits(cfg, other, toks), place)


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
        "hf_checkpoint": path, "tokenizer": "ids", "model": {"type": "zosipel"}, "prompts": [" ".join(map(str, prompt))], "max_new_tokens": 12,
        "n_rounds": 1, "stop_sequence": None, "temperature": 0.0, "engine": {"max_seqs": 2, "page_size": 8, "max_pages_per_seq": 6, "compute_dtype": "float32"},
        "trainer": {"require_accelerator": False, "tracker": {"type": "noop"}, "log_dir": str(tmp_path), "mp": "f32"}}))
    out = capsys.readouterr().out
    toks = list(prompt)
    for _ in range(12):
        toks.append(int(O.logits(cfg, W, toks)[-1].argmax()))
    want = [t for t in toks[21:] if t != cfg["vocab"] - 1]  # the command drops the padding token
    got = out.split("Generated text for 0", 1)[1].split(":", 1)[1].split("\n")[0].split()
    assert [int(t) for t in got] == want
