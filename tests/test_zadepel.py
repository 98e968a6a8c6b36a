"""Zadepel through the framework (registry, checkpoint loading, engine, scheduler, trace replay) against ``zadepel_oracle``: on the CPU
in fp32, and on a B200 in fp32 and bf16."""
import dataclasses
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import zadepel_oracle as O
from levanter_b200.compat.hf_checkpoints import HFCheckpointConverter
from levanter_b200.inference.engine import Request
from levanter_b200.inference.jit_scheduler import SeqDecodingParams
from levanter_b200.layers.attention import AttentionMask
from levanter_b200.layers.recurrence import SlotStateCache
from levanter_b200.models.lm_model import LmConfig, LmExample
from levanter_b200.models.zadepel import ZadepelConfig, ZadepelLayerConfig, ZadepelLMHeadModel
from test_fedolorn import PLACES, ROOT, _cuts, _engine, _feed, _load, _tokens


def _attn(heads, kv, dim, vdim, scale, dims, base, v_mix=True):
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, rot=dict(base=base, dims=dims), v_mix=v_mix))


def _latent(heads, dim, rot_dim, vdim, rank, window, scale, base):
    return dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=rank, scale=scale, mask={"size": window},
                                                    rot=dict(base=base, dims=rot_dim)))


def _gru(width):
    return dict(type="mingru", mixer=dict(width=width))


def _config(name):
    """Small models that differ in every size and constant, from each other and from layer to layer."""
    if name == "mixed":  # a plain attention layer comes before the first one that mixes values
        layers = [(_gru(40), 56), (_attn(6, 3, 24, 16, 0.3, 8, 300.0, False), 48), (_latent(5, 24, 8, 32, 40, 20, 0.25, 900.0), None),
                  (_attn(4, 2, 32, 24, 0.35, 32, 5000.0), 64), (_latent(3, 16, 16, 8, 24, 7, 0.3, 50.0), 40), (_attn(8, 2, 16, 24, 0.4, 16, 200.0), 72),
                  (_gru(104), None)]
        cfg = dict(architecture="Zadepel", vocab=83, width=72, norm={"eps": 0.01})
    elif name == "odd":  # sizes that are not multiples of 8
        layers = [(_latent(3, 10, 6, 14, 18, 33, 0.37, 70.0), 22), (_attn(4, 1, 14, 10, 0.5, 6, 40.0), None), (_gru(21), 30),
                  (_attn(6, 3, 10, 18, 0.4, 10, 90.0, False), 18), (_attn(2, 1, 18, 10, 0.3, 18, 1000.0), 26)]
        cfg = dict(architecture="Zadepel", vocab=45, width=50, norm={"eps": 1e-4})
    else:  # one of everything, and a window of one token
        layers = [(_attn(1, 1, 8, 8, 1.0, 2, 10.0), 8), (_latent(1, 8, 2, 8, 8, 1, 1.0, 10.0), 8), (_gru(8), 8)]
        cfg = dict(architecture="Zadepel", vocab=24, width=16, norm={"eps": 1e-6})
    return dict(cfg, layers=[dict(l, mlp=None if ff is None else dict(kind="dense", ff=ff)) for l, ff in layers])


NAMES = ["mixed", "odd", "ones"]


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
    """Row by row.  The heads are sharp on purpose, so bf16 rounding alone moves a few rows far; a fault moves a row by about 1."""
    got, want = torch.as_tensor(got).double().cpu(), want.double()
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    if place[1] == torch.float32:
        assert float(err.max()) < 1e-4, (what, int(err.argmax()), float(err.max()))
    else:
        assert float(err.median()) < 0.06 and float((err > 0.15).double().mean()) <= 0.1 and float(err.max()) < 0.5, (what, int(err.argmax()), err)


def test_registry_config_and_checkpoint_names(checkpoint, tmp_path):
    cfg, W, path = checkpoint("mixed")
    assert LmConfig.get_known_choices()["zadepel"] is ZadepelConfig
    conv = HFCheckpointConverter.from_hf(path)
    c = conv.config_from_hf_checkpoint(path)
    assert isinstance(c, ZadepelConfig) and c.num_layers == 7 and c.layers[2].intermediate_dim is None and c.layers[4].sliding_window == 7
    assert c.to_hf_config(83) == cfg
    m = _load(path, ("cpu", torch.bfloat16))
    assert isinstance(m, ZadepelLMHeadModel) and m.vocab_size == 83
    W = {k: v for k, v in W.items() if k != "l1.mix.vmix"}  # a layer that mixes nothing has no such number
    assert sum(p.numel() for p in m.parameters()) == sum(t.numel() for t in W.values()) == c.total_trainable_params(83)
    assert c.flops_per_token(83) > 0
    conv.save_pretrained(m, str(tmp_path / "out"), save_tokenizer=False)
    from safetensors.torch import load_file

    back = load_file(str(tmp_path / "out" / "model.safetensors"))
    assert back.keys() == W.keys() and all(torch.equal(back[k], W[k]) for k in W)
    assert json.loads((tmp_path / "out" / "config.json").read_text())["layers"] == cfg["layers"]


def test_config_from_yaml_and_rejected_configs():
    from levanter_b200 import config as lev_config

    c = lev_config.decode(LmConfig, {"type": "zadepel", "hidden_dim": 32, "layers": [
        {"mixer": "attention", "num_heads": 2, "num_kv_heads": 1, "head_dim": 8, "v_head_dim": 8, "rotary_dim": 4, "intermediate_dim": 16},
        {"mixer": "mingru", "width": 24, "intermediate_dim": None},
        {"mixer": "latent_attention", "num_heads": 2, "head_dim": 8, "v_head_dim": 8, "rotary_dim": 4, "kv_lora_rank": 8, "sliding_window": 3,
         "intermediate_dim": 16}]})
    assert isinstance(c, ZadepelConfig) and all(isinstance(l, ZadepelLayerConfig) for l in c.layers) and c.layers[2].sliding_window == 3
    m = c.build(11, seed=0)
    assert m(torch.arange(5)[None]).shape == (1, 5, 11)
    with pytest.raises(ValueError):
        m.initial_cache(4, 8)  # recurrent state needs the number of slots
    for bad in (dict(num_heads=3, num_kv_heads=2), dict(mixer="other"), dict(rotary_dim=200), dict(rotary_dim=7), dict(sliding_window=0)):
        with pytest.raises(ValueError):
            ZadepelLayerConfig(**bad)
    with pytest.raises(ValueError):
        ZadepelConfig(layers=(ZadepelLayerConfig(), ZadepelLayerConfig(v_head_dim=64)))
    for change in (lambda l: l.update(type="other"), lambda l: l["mlp"].update(kind="other")):
        entry = _config("mixed")
        change(entry["layers"][1])
        with pytest.raises(ValueError):
            ZadepelConfig.from_hf_config(entry)


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
    sequences restart their states and windows."""
    cfg, W, path = checkpoint("mixed")
    m = _load(path, ("cpu", torch.float32))
    a, b = _tokens(30, 83, 1), _tokens(45, 83, 2)
    seg = torch.tensor([0] * 30 + [1] * 45)
    ex = LmExample.causal(torch.tensor(a + b), segment_ids=seg)
    with torch.no_grad():
        got = m(ex.tokens[None], dataclasses.replace(ex.attn_mask, segment_ids=(seg[None], seg[None])))[0]
    _close(got, torch.cat([O.logits(cfg, W, a), O.logits(cfg, W, b)]), ("cpu", torch.float32))
    toks = torch.tensor(a)
    ref = torch.randn(30, 83, generator=torch.Generator().manual_seed(0), dtype=torch.float64)
    (m(toks[None])[0].double() * ref).sum().backward()
    kept = {n: p.grad.clone() for n, p in m.named_parameters() if p.grad is not None}
    m.zero_grad()
    m.train()
    (m(toks[None])[0].double() * ref).sum().backward()
    params = dict(m.named_parameters())
    assert {n for n, p in params.items() if p.grad is None} == {"transformer.layers.3.mixer.value_mix"}  # the first mixing layer's is unused
    assert all(torch.allclose(params[n].grad, g, rtol=1e-4, atol=1e-4 * float(g.abs().max())) for n, g in kept.items())
    for pname in ("transformer.layers.0.mixer.z_proj.weight", "transformer.layers.0.mixer.x_proj.bias", "transformer.layers.2.mixer.kv_b_proj.weight",
                  "transformer.layers.3.mixer.v_proj.weight", "transformer.layers.5.mixer.value_mix", "transformer.layers.5.mixer.temperature",
                  "transformer.layers.4.post_mlp_layernorm.weight", "embeddings.token_embeddings.weight"):
        d = torch.randn(params[pname].shape, generator=torch.Generator().manual_seed(1), dtype=torch.float64)
        vals = []
        for sgn in (1, -1):
            W2 = {k: v.double() for k, v in W.items()}
            for n, view, shape in m.hf_tensor_parts(pname, d):
                W2[n] = W2[n] + sgn * 1e-5 * view.reshape(shape)
            vals.append((O.logits(cfg, W2, a) * ref).sum())
        fd = float((vals[0] - vals[1]) / 2e-5)
        got = float((params[pname].grad.double() * d).sum())
        assert abs(got - fd) <= 2e-3 * max(abs(fd), 1.0), (pname, got, fd)


# ------------------------------------------------------------------------------------------------ serving
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("place", PLACES)
def test_prompt_portions_and_token_by_token(checkpoint, name, place):
    """The same sequence in one step, in portions of several sizes, and decoded one token at a time, across page and window borders
    of every layer; each form on pages and state slots that the previous one gave back."""
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
    small that every page and slot is used several times."""
    cfg, W, path = checkpoint("mixed")
    m = _load(path, place)
    eng = _engine(m, place, max_seqs=4, max_pages=60)
    lens = {"a": 1, "b": 66, "c": 19, "d": 41}
    full = {k: _tokens(n + 25, cfg["vocab"], i) for i, (k, n) in enumerate(lens.items())}
    want = {k: O.logits(cfg, W, t) for k, t in full.items()}
    for order in ("abcd", "dbca"):  # the second time every request gets a slot that held another one's state
        got, slots = _feed(eng, [[(k, full[k][:lens[k]]) for k in order]] + [[(k, full[k][lens[k] + i:lens[k] + i + 1]) for k in order] for i in range(25)])
        for k in lens:
            _close(got[k], want[k], place, k)
        eng.close_sequences(slots.values())
    # ragged: one decodes, one goes on with a portion, one starts
    s = {k: eng.open_sequence() for k in "abc"}
    eng.forward_packed([(s["a"], full["a"][:5]), (s["b"], full["b"][:30])], [])
    rows = eng.forward_packed([(s["a"], full["a"][5:6]), (s["b"], full["b"][30:43]), (s["c"], full["c"][:22])], list(range(36))).float().cpu()
    for part, k, lo, hi in ((rows[:1], "a", 5, 6), (rows[1:14], "b", 30, 43), (rows[14:], "c", 0, 22)):
        _close(part, want[k][lo:hi], place, k)
    # a request ends, its slot goes to a new one, the others go on
    eng.close_sequences([s["a"]])
    s["d"] = eng.open_sequence()
    assert s["d"] == s["a"]
    rows = eng.forward_packed([(s["d"], full["d"][:2]), (s["b"], full["b"][43:44])], [0, 1, 2]).float().cpu()
    _close(rows[:2], want["d"][:2], place, "d")
    _close(rows[2:], want["b"][43:44], place, "b")


@pytest.mark.parametrize("place", PLACES)
def test_greedy_generation_through_the_scheduler(checkpoint, place):
    """More requests than slots, clones (pages and recurrent state), early stops, long decoding over several windows."""
    cfg, W, path = checkpoint("mixed")
    m = _load(path, place)
    eng = _engine(m, place, max_seqs=3, pages_per_seq=40, max_pages=110, max_rounds=5, use_cuda_graph=place[0] == "cuda")
    assert sum(isinstance(c, SlotStateCache) for c in eng.gen_state.cache) == 2
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
                    assert float(gap.max()) < 0.2, (i, gap)
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
    for s, rows in wanted.items():
        got = torch.from_numpy(np.fromfile(tmp_path / f"{s}.f32", dtype="<f4").reshape(len(rows), cfg["vocab"]))
        _close(got, torch.stack([want[k][p] for k, p in rows]), place, s)


@pytest.mark.parametrize("place", PLACES)
def test_weights_that_change_after_serving(checkpoint, place):
    """Derived weights (joint projections, whole-key products) follow their parameters: the same engine after a load of other weights."""
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
        "hf_checkpoint": path, "tokenizer": "ids", "model": {"type": "zadepel"}, "prompts": [" ".join(map(str, prompt))], "max_new_tokens": 12,
        "n_rounds": 1, "stop_sequence": None, "temperature": 0.0, "engine": {"max_seqs": 2, "page_size": 8, "max_pages_per_seq": 6, "compute_dtype": "float32"},
        "trainer": {"require_accelerator": False, "tracker": {"type": "noop"}, "log_dir": str(tmp_path), "mp": "f32"}}))
    out = capsys.readouterr().out
    toks = list(prompt)
    for _ in range(12):
        toks.append(int(O.logits(cfg, W, toks)[-1].argmax()))
    want = [t for t in toks[21:] if t != cfg["vocab"] - 1]  # the command drops the padding token
    got = out.split("Generated text for 0", 1)[1].split(":", 1)[1].split("\n")[0].split()
    assert [int(t) for t in got] == want


@pytest.mark.parametrize("place", PLACES)
def test_windowed_mistral_decodes_in_its_window(place):
    """A family that had its window in training and prefill only: decoding through the cache agrees with the whole forward."""
    from levanter_b200.models.mistral import MistralConfig

    c = MistralConfig(seq_len=128, hidden_dim=64, intermediate_dim=96, num_layers=2, num_heads=4, num_kv_heads=2, head_dim=32, sliding_window=5, apply_sliding_window=True,
                      initializer_range=0.2)
    torch.manual_seed(0)
    m = c.build(40, seed=0).to(place[0], place[1]).eval()
    toks = _tokens(37, 40, 4)
    with torch.no_grad():
        want = m(torch.tensor([toks], device=place[0]), AttentionMask.causal())[0].double().cpu()
    got, _ = _feed(_engine(m, place), [[("a", toks[:11])]] + [[("a", [t])] for t in toks[11:]])
    _close(got["a"], want, place)
