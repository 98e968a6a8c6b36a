"""Mumizen through the framework (registry, checkpoint loading, engine, scheduler, trace replay) against ``mumizen_oracle``: on the CPU
in fp32, and on a B200 in fp32 and bf16."""
import dataclasses
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import mumizen_oracle as O
from levanter_b200.compat.hf_checkpoints import HFCheckpointConverter
from levanter_b200.inference.engine import Request
from levanter_b200.inference.jit_scheduler import SeqDecodingParams
from levanter_b200.layers.normalization import GroupedRmsNormConfig, LayerNormConfigBase
from levanter_b200.layers.rotary import DefaultRotaryEmbeddingsConfig, PartialYarnRotaryEmbeddingsConfig
from levanter_b200.models.lm_model import LmConfig, LmExample
from levanter_b200.models.mumizen import MumizenConfig, MumizenLayerConfig, MumizenLMHeadModel
from test_fedolorn import PLACES, ROOT, _cuts, _engine, _feed, _load, _tokens


def _linear(kind, heads, dim, vdim, decay):
    return dict(type=kind, mixer=dict(heads=heads, dim=dim, vdim=vdim, decay=list(decay)))


def _latent(heads, dim, rot_dim, vdim, q_rank, rank, scale, base, yarn=None, kv_from=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=rank, scale=scale, rot=dict(base=base, dims=rot_dim))
    if yarn is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="latent_attention", mixer=m)


def _dense(ff, limit):
    return dict(kind="dense", ff=ff, limit=limit)


def _moe(ff, limit, experts, top, shared=None):
    f = dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top))
    return f if shared is None else dict(f, shared=dict(zip(("ff", "limit"), shared)))


def _whole(vocab, width, eps, groups, layers):
    return dict(architecture="Mumizen", vocab=vocab, width=width, norm=dict(eps=eps, groups=groups), layers=[dict(l, mlp=f) for l, f in layers])


YARN = (8.0, 24, 4.0, 0.5)


def _config(name):
    """Small models that differ in every size and constant, from each other and from layer to layer."""
    if name == "mixed":  # two layers that keep latents and three that read them, one of them right after and one over others; all feed-forwards
        layers = [(_latent(5, 24, 16, 32, 56, 40, 0.25, 300.0, YARN), _moe(24, 0.75, 10, 3, (40, 2.0))),
                  (_linear("retention", 3, 16, 40, (0.5, 0.97, 1.0)), _dense(56, 0.5)),
                  (_latent(3, 40, 16, 16, 24, 40, 0.2, 300.0, YARN, kv_from=0), None),
                  (_linear("lightning", 4, 24, 16, (0.2, 0.9, 0.99, 0.9995)), _moe(16, 1.5, 6, 2)),
                  (_latent(2, 16, 8, 48, 40, 72, 0.3, 5000.0), _dense(24, 3.0)),
                  (_latent(6, 8, 16, 24, 32, 40, 0.35, 300.0, YARN, kv_from=0), _moe(8, 0.3, 9, 4, (16, 0.6))),
                  (_linear("lightning", 1, 72, 80, (0.95,)), None),
                  (_latent(2, 24, 8, 8, 16, 72, 0.15, 5000.0, kv_from=4), _dense(40, 1.25))]
        return _whole(83, 72, 0.01, 3, layers)
    if name == "odd":  # sizes that are not multiples of 8 (groups of 10), linear attention in the first and last layer
        layers = [(_linear("lightning", 3, 10, 14, (0.7, 0.99, 0.0)), _dense(22, 0.8)),
                  (_latent(3, 14, 6, 10, 22, 18, 0.37, 40.0, (2.0, 100, 8.0, 2.0)), _moe(10, 0.9, 7, 3, (6, 0.4))),
                  (_latent(4, 10, 6, 18, 9, 18, 0.3, 40.0, (2.0, 100, 8.0, 2.0), kv_from=1), _dense(13, 2.0)),
                  (_linear("retention", 5, 6, 9, (0.3, 0.6, 0.9, 0.99, 0.999)), _moe(14, 1.1, 6, 2))]
        return _whole(45, 50, 1e-4, 5, layers)
    if name == "linear":  # no pages at all; one group
        layers = [(_linear("retention", 2, 136, 24, (0.99, 0.6)), _dense(48, 1.0)), (_linear("lightning", 2, 32, 64, (0.9, 0.9999)), _moe(32, 2.5, 5, 1, (24, 1.0)))]
        return _whole(61, 64, 1e-5, 1, layers)
    # one of everything: one head, one expert, one element per group, a rotation of one pair
    layers = [(_latent(1, 8, 2, 8, 8, 8, 1.0, 10.0, (1.0, 16, 2.0, 1.0)), None), (_linear("retention", 1, 8, 8, (1.0,)), _moe(8, 1.0, 1, 1, (8, 1.0))),
              (_linear("lightning", 1, 1, 1, (0.5,)), _dense(1, 1.0))]
    return _whole(24, 16, 0.05, 16, layers)  # (a group of one element is its sign: the epsilon keeps it from jumping)


NAMES = ["mixed", "odd", "linear", "ones"]


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
        assert float(err.max()) < 2e-4, (what, int(err.argmax()), float(err.max()))
    else:
        assert float(err.median()) < 0.05 and float((err > 0.15).double().mean()) <= 0.15, (what, int(err.argmax()), err)


def test_registry_config_and_checkpoint_names(checkpoint, tmp_path):
    cfg, W, path = checkpoint("mixed")
    assert LmConfig.get_known_choices()["mumizen"] is MumizenConfig
    assert LayerNormConfigBase.get_known_choices()["rms_grouped"] is GroupedRmsNormConfig
    conv = HFCheckpointConverter.from_hf(path)
    c = conv.config_from_hf_checkpoint(path)
    assert isinstance(c, MumizenConfig) and c.num_layers == 8 and c.layers[2].intermediate_dim is None and c.layers[5].kv_from == 0 and c.norm_groups == 3
    assert isinstance(c.layers[0].rope, PartialYarnRotaryEmbeddingsConfig) and isinstance(c.layers[4].rope, DefaultRotaryEmbeddingsConfig)
    assert c.to_hf_config(83) == cfg
    m = _load(path, ("cpu", torch.bfloat16))
    assert isinstance(m, MumizenLMHeadModel) and m.vocab_size == 83
    assert sum(p.numel() for p in m.parameters()) == sum(t.numel() for t in W.values()) == c.total_trainable_params(83)
    assert c.flops_per_token(83) > 0
    cache = m.initial_cache(4, 8, 3)
    assert [x.mixer is None for x in cache] == [False, False, True, False, False, True, False, True]  # shared latents are kept once
    assert cache[1].mixer.state.shape == (3, 3, 16, 40) and cache[1].mixer.state.dtype == torch.float32 and cache[7].shift.state.shape == (3, 72)
    conv.save_pretrained(m, str(tmp_path / "out"), save_tokenizer=False)
    from safetensors.torch import load_file

    back = load_file(str(tmp_path / "out" / "model.safetensors"))
    assert back.keys() == W.keys() and all(torch.equal(back[k], W[k]) for k in W)
    assert json.loads((tmp_path / "out" / "config.json").read_text())["layers"] == cfg["layers"]
    for name in ("odd", "linear", "ones"):
        assert MumizenConfig.from_hf_config(_config(name)).to_hf_config(_config(name)["vocab"]) == _config(name)


def test_config_from_yaml_and_rejected_configs():
    from levanter_b200 import config as lev_config

    c = lev_config.decode(LmConfig, {"type": "mumizen", "hidden_dim": 32, "norm_groups": 2, "layers": [
        {"mixer": "retention", "num_heads": 2, "head_dim": 8, "v_head_dim": 8, "decay": [0.5, 0.9], "intermediate_dim": 16, "limit": 2.0},
        {"mixer": "latent_attention", "num_heads": 2, "head_dim": 8, "v_head_dim": 8, "rotary_dim": 4, "q_lora_rank": 8, "kv_lora_rank": 8,
         "rope": {"type": "yarn_partial", "theta": 100.0, "factor": 2.0}, "intermediate_dim": 8, "num_experts": 4, "num_experts_per_tok": 2},
        {"mixer": "lightning", "num_heads": 1, "head_dim": 8, "v_head_dim": 8, "decay": [0.9], "intermediate_dim": None}]})
    assert isinstance(c, MumizenConfig) and all(isinstance(l, MumizenLayerConfig) for l in c.layers) and c.layers[1].rope.factor == 2.0
    assert c.layers[0].decay == (0.5, 0.9)
    m = c.build(11, seed=0)
    assert m(torch.arange(5)[None]).shape == (1, 5, 11)
    for bad in (dict(mixer="other"), dict(decay=(0.5,)), dict(decay=(0.5,) * 16, num_experts=4, num_experts_per_tok=5), dict(mixer="latent_attention", rotary_dim=7),
                dict(mixer="latent_attention", rope=DefaultRotaryEmbeddingsConfig(rotary_dim=32)), dict(mixer="latent_attention", kv_from=-1)):
        with pytest.raises(ValueError):
            MumizenLayerConfig(**bad)
    lin, own = MumizenLayerConfig(decay=(0.5,) * 16), MumizenLayerConfig(mixer="latent_attention")
    reads = dataclasses.replace(own, kv_from=0)
    MumizenConfig(layers=(own, lin, reads))
    for layers in ((), (reads,), (lin, reads), (own, reads, dataclasses.replace(own, kv_from=1)), (own, dataclasses.replace(reads, kv_lora_rank=256)),
                   (own, dataclasses.replace(reads, rope=DefaultRotaryEmbeddingsConfig(theta=5.0))), (own, dataclasses.replace(own, kv_from=1))):
        with pytest.raises(ValueError):
            MumizenConfig(layers=layers)
    with pytest.raises(ValueError):
        MumizenConfig(norm_groups=3, layers=(own,))
    for change in (lambda l: l.update(type="other"), lambda l: l["mlp"].update(kind="other"), lambda l: l["mixer"]["rot"].update(dims=8)):
        entry = _config("mixed")
        change(entry["layers"][0])
        with pytest.raises(ValueError):
            MumizenConfig.from_hf_config(entry)


@pytest.mark.parametrize("segments", [None, [0, 0, 0, 1, 1, 5, 5, 5, 5, 5, 2] + [3] * 60 + [4] * 9])
@pytest.mark.parametrize("chunk", [1, 4, 64, 100])
def test_linear_attention_by_chunks(segments, chunk):
    """The differentiable form: chunks of several sizes against the recurrence, also when sequences begin inside chunks."""
    from levanter_b200.ops.linear_attention import fixed_decay_attention

    g = torch.Generator().manual_seed(0)
    n, decay = 80, (0.0, 0.3, 0.99, 1.0)
    q, k, v = (torch.randn(n, 4, d, generator=g, dtype=torch.float64) for d in (6, 6, 10))
    seg = torch.tensor(segments or [0] * n)
    got = fixed_decay_attention(q[None], k[None], v[None], torch.tensor(decay), None if segments is None else seg[None], chunk)[0]
    cuts = [0] + (1 + (seg[1:] != seg[:-1]).nonzero()[:, 0]).tolist() + [n]
    want = torch.cat([O.fixed_decay_attention(q[a:b], k[a:b], v[a:b], decay) for a, b in zip(cuts, cuts[1:])])
    assert torch.allclose(got.double(), want, atol=1e-4)


def test_grouped_norm_token_shift_and_clamped_gate():
    """The small pieces in their differentiable forms."""
    from levanter_b200.nn import GroupedRmsNorm
    from levanter_b200.ops.depth_stream import shift_tokens
    from levanter_b200.ops.glu import ClampedGlu, gated_activation

    g = torch.Generator().manual_seed(0)
    x, w, mu = torch.randn(9, 24, generator=g), torch.randn(24, generator=g), torch.rand(24, generator=g)
    for groups in (1, 3, 24):
        norm = GroupedRmsNorm(24, groups, eps=0.1)
        with torch.no_grad():
            norm.weight.copy_(w)
            for got in (norm(x), norm.from_stream(x)):
                assert torch.allclose(got.double(), O.grouped_rms_norm(x.double(), w.double(), groups, 0.1), atol=1e-5)
    assert torch.allclose(shift_tokens(x[None], mu)[0].double(), O.shift_tokens(x.double(), mu.double()), atol=1e-6)
    starts = torch.zeros(1, 9, dtype=torch.bool)
    starts[0, [0, 4]] = True
    want = torch.cat([O.shift_tokens(x[:4].double(), mu.double()), O.shift_tokens(x[4:].double(), mu.double())])
    assert torch.allclose(shift_tokens(x[None], mu, starts)[0].double(), want, atol=1e-6)
    gate, up = 3 * torch.randn(50, generator=g, dtype=torch.float64), 3 * torch.randn(50, generator=g, dtype=torch.float64)
    for limit in (0.3, 1.0, 7.0):
        assert torch.allclose(gated_activation(gate.float(), up.float(), ClampedGlu(limit)).double(), O.clamped_gate(gate, up, limit), atol=1e-5)
    with pytest.raises(ValueError):
        GroupedRmsNorm(24, 5)


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
    sequences restart their states, shifts and positions."""
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
    for pname in ("transformer.layers.0.mixer.kv_a_proj.weight", "transformer.layers.0.mixer.kv_a_norm.weight", "transformer.layers.2.mixer.kv_b_proj.weight",
                  "transformer.layers.5.mixer.q_a_proj.weight", "transformer.layers.7.mixer.g_proj.weight", "transformer.layers.1.mixer.k_proj.weight",
                  "transformer.layers.3.mixer.v_proj.weight", "transformer.layers.6.mixer.o_norm.weight", "transformer.layers.3.shift",
                  "transformer.layers.4.depth_weights", "transformer.layers.0.mlp.experts.gate_up", "transformer.layers.0.mlp.router.bias",
                  "transformer.layers.0.mlp.shared.up_proj.weight", "transformer.layers.1.mlp.gate_proj.weight",
                  "transformer.layers.1.post_mixer_layernorm.weight", "transformer.layers.6.input_layernorm.weight", "lm_head.weight"):
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
    """The same sequence in one step, in portions of several sizes, and decoded one token at a time, across page and chunk borders;
    each form on pages and slots that the previous one gave back."""
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
    """More requests than slots, clones, early stops, long decoding."""
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
    """Derived weights (joint projections, whole-key products) follow their parameters: the same engine after a load of other
    weights."""
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
        "hf_checkpoint": path, "tokenizer": "ids", "model": {"type": "mumizen"}, "prompts": [" ".join(map(str, prompt))], "max_new_tokens": 12,
        "n_rounds": 1, "stop_sequence": None, "temperature": 0.0, "engine": {"max_seqs": 2, "page_size": 8, "max_pages_per_seq": 6, "compute_dtype": "float32"},
        "trainer": {"require_accelerator": False, "tracker": {"type": "noop"}, "log_dir": str(tmp_path), "mp": "f32"}}))
    out = capsys.readouterr().out
    toks = list(prompt)
    for _ in range(12):
        toks.append(int(O.logits(cfg, W, toks)[-1].argmax()))
    want = [t for t in toks[21:] if t != cfg["vocab"] - 1]  # the command drops the padding token
    got = out.split("Generated text for 0", 1)[1].split(":", 1)[1].split("\n")[0].split()
    assert [int(t) for t in got] == want
