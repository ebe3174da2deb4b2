"""Bumulix without a GPU: its configuration and weight plan, and the engine's host side (several
residual streams, paged stores with windows and with latents, layers that run with another
layer's tensors and storage of their own, slots, pages, batches, the generation loop) on the
torch-CPU stand-in of the kernel library, against the plain implementation."""
import copy
import io
import json

import pytest
import torch

import bumulix_models as BM
import plain_bumulix as PB
from nimbus_infer_rs_b200 import Engine, SamplingParams
from nimbus_infer_rs_b200.config import BumulixConfig, ConfigError
from nimbus_infer_rs_b200.config.registry import load_config, resolve_architecture
from nimbus_infer_rs_b200.engine.spec import LayerSpec, ModelSpec
from nimbus_infer_rs_b200.parts.base import KVRequest, PartSpec
from nimbus_infer_rs_b200.weights.loader import WeightError

NAMES = list(BM.CONFIGS)


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("bumulix")
    return {n: BM.make(root, n) for n in NAMES}


def _tokens(vocab, n, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def _close(got, ref, tol=3e-5):
    got, ref = got.double(), ref.double()
    assert got.shape == ref.shape
    assert float((got - ref).abs().max()) <= tol * float(ref.abs().max())


def _engine(models, name, **kw):
    kw.setdefault("cache_tokens", 1024)
    return Engine.load(models[name][0], dtype="float32", device="cpu", **kw)


def test_config_is_read_and_recognised(models):
    folder, _, _ = models["A"]
    arch, typed = load_config(folder)
    assert arch.name == "bumulix" and isinstance(typed, BumulixConfig)
    assert resolve_architecture({"architecture": "bumulix"}).name == "bumulix"
    assert (typed.vocab_size, typed.width, typed.norm_eps) == (211, 56, 3e-5)
    assert (typed.streams, typed.residual_mult, typed.logit_softcap) == (3, 0.7, 12.0)
    a = typed.layers[0].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.diff, a.mask_size) == (4, 2, 12, 20, 0.3, 0.4, 9)
    b = typed.layers[1].mixer
    assert (b.heads, b.dim, b.rot_dim, b.vdim, b.kv_rank, b.q_rank) == (3, 14, 10, 12, 20, 18)
    assert b.rot.base == 500.0 and b.rot.scaling() == {"factor": 4.0, "original": 64.0, "fast": 8.0, "slow": 0.5}
    assert typed.layers[2].weights_of == 1 and typed.owner(2) == 1 and typed.layers[3].mlp is None
    for n in NAMES:
        c = BumulixConfig.from_json(BM.CONFIGS[n])
        assert BumulixConfig.from_json(c.to_json()) == c
    # what is left out is absent
    e = BumulixConfig.from_json(BM.CONFIGS["E"])
    assert e.streams is None and e.layers[2].mixer.mask_size == 0
    c = BumulixConfig.from_json(BM.CONFIGS["C"])
    assert c.residual_mult == 1.0 and c.logit_softcap == 0.0 and c.layers[1].mixer.rot.scaling() is None
    # sizes that follow from others
    short = copy.deepcopy(BM.CONFIGS["C"])
    for key in ("kv_heads", "vdim"):
        del short["layers"][0]["mixer"][key]
    m = BumulixConfig.from_json(short).layers[0].mixer
    assert m.kv_heads == m.heads and m.vdim == 2 * m.dim


def test_config_errors_name_every_bad_key():
    bad = copy.deepcopy(BM.CONFIGS["A"])
    bad["layers"][0]["mixer"]["heads"] = 3                     # no multiple of kv_heads
    bad["layers"][1]["mixer"]["rot"]["dims"] = 12              # more than rot_dim
    del bad["layers"][1]["mixer"]["rot"]["scaling"]["fast"]
    bad["layers"][2]["mixer"] = {"heads": 3}
    bad["layers"][3]["type"] = "windowed"
    bad["layers"][0]["mlp"] = {"kind": "sparse"}
    bad["layers"][0]["mixer"].pop("diff")
    bad["streams"] = 9
    del bad["norm"]
    with pytest.raises(ConfigError) as e:
        BumulixConfig.from_json(bad)
    msg = str(e.value)
    for piece in ("kv_heads", "rot.dims", "scaling.fast", "kv_rank", "windowed", "sparse", "diff",
                  "config.streams", "norm.eps"):
        assert piece in msg, piece
    other = copy.deepcopy(BM.CONFIGS["A"])
    other["layers"][2]["mixer"] = dict(other["layers"][2]["mixer"], scale=0.31)
    with pytest.raises(ConfigError):
        BumulixConfig.from_json(other)
    circle = copy.deepcopy(BM.CONFIGS["A"])
    circle["layers"][1]["weights_of"] = 2
    with pytest.raises(ConfigError):
        BumulixConfig.from_json(circle)


def test_weight_errors_are_listed_together(models, tmp_path):
    _, cfg, tensors = models["A"]
    t = dict(tensors)
    del t["l1.mix.dq.norm"], t["l0.hc2.mix"]
    t["l0.mix.lq2"] = torch.zeros(13)
    t["l2.norm1"] = torch.zeros(56)          # a layer without tensors of its own has none
    t["l3.hc2.in"] = torch.zeros(3)          # stands around a feed-forward that is not there
    folder = BM.write_model(tmp_path / "bad", cfg, t)
    with pytest.raises(WeightError) as e:
        Engine.load(folder, dtype="float32", device="cpu")
    assert e.value.missing == ["l0.hc2.mix", "l1.mix.dq.norm"] and e.value.unexpected == ["l2.norm1"]
    assert any("lq2" in w for w in e.value.wrong_shape)


def test_streams_and_arrangements_must_fit():
    norm = PartSpec("rmsnorm", {"width": 8, "eps": 1e-5})
    mixer = PartSpec("causal_attention", {"width": 8, "n_heads": 1, "n_kv_heads": 1, "head_dim": 8, "scale": 1.0})

    def spec(block, streams):
        return ModelSpec("x", 10, 8, None, PartSpec("none"),
                         (LayerSpec(mixer, None, norm, None, block=block),), norm, streams=streams)
    with pytest.raises(ValueError, match="residual streams"):
        spec(PartSpec("pre_norm"), 2).validate()
    with pytest.raises(ValueError, match="residual streams"):
        spec(PartSpec("hyper_connections", {"width": 8, "streams": 3}), 2).validate()
    spec(PartSpec("hyper_connections", {"width": 8, "streams": 2}), 2).validate()


@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_and_token_by_token(models, cpu_backend, name):
    _, cfg, P = models[name]
    e = _engine(models, name)
    for n in (1, 2, 37, 80):
        toks = _tokens(cfg["vocab"], n, n)
        ref = PB.logits(toks, P, cfg)
        s = e.alloc_slot()
        _close(e.step([(s, toks, list(range(n)))]), ref)
        e.free_slot(s)
        s = e.alloc_slot()
        _close(torch.cat([e.step([(s, [t], [0])]) for t in toks]), ref)
        e.free_slot(s)


def test_layer_by_layer(models, cpu_backend):
    """The sum of the streams after every layer run (tensors that run twice count each time)."""
    _, cfg, P = models["A"]
    e = _engine(models, "A")
    assert e.model.run_order == (0, 1, 1, 2, 0) and len(e.model.layers) == 3
    snaps = []
    for l in e.model.layers:
        f = l.block.forward

        def tapped(ctx, x, layer, f=f):
            f(ctx, x, layer)
            snaps.append((x.view(x.shape[0], 3, -1).sum(1) if ctx.streams_sum is None
                          else ctx.streams_sum).clone())
        l.block.forward = tapped
    toks = _tokens(211, 50, 5)
    e.step([(e.alloc_slot(), toks, [0])])
    ref = PB.hidden_states(toks, P, cfg)
    assert len(snaps) == ref.shape[0] == 5
    for got, want in zip(snaps, ref):
        _close(got[:50], want)


@pytest.mark.parametrize("name", ["A", "D", "E"])
def test_portions_down_to_two_tokens(models, cpu_backend, name):
    _, cfg, P = models[name]
    e = _engine(models, name)
    toks = _tokens(cfg["vocab"], 150, 3)
    s, at, outs = e.alloc_slot(), 0, []
    for size in (2, 61, 1, 2, 64, 3, 17):
        outs.append(e.step([(s, toks[at:at + size], list(range(size)))]))
        at += size
    _close(torch.cat(outs), PB.logits(toks, P, cfg))


def test_unequal_batch_on_slots_and_pages_used_again(models, cpu_backend):
    _, cfg, P = models["A"]
    e = _engine(models, "A", cache_tokens=5 * 64, n_slots=3)
    for turn, lens in enumerate(((100, 5, 66), (1, 90, 30))):
        seqs = [_tokens(211, n, 17 * turn + i) for i, n in enumerate(lens)]
        heads = [max(1, n - 3 - i) for i, n in enumerate(lens)]
        slots = [e.alloc_slot() for _ in lens]
        got = {i: [] for i in range(3)}
        out = e.step([(slots[i], seqs[i][:heads[i]], [heads[i] - 1]) for i in range(3)])
        for i in range(3):
            got[i].append(out[i])
        k = 0
        while True:
            live = [i for i in range(3) if heads[i] + k < lens[i]]
            if not live:
                break
            out = e.step([(slots[i], [seqs[i][heads[i] + k]], [0]) for i in live])
            for j, i in enumerate(live):
                got[i].append(out[j])
            k += 1
        for i in range(3):
            _close(torch.stack(got[i]), PB.logits(seqs[i], P, cfg)[heads[i] - 1:])
            e.free_slot(slots[i])
    assert all(g.pool.n_free == g.pool.n_pages for g in e.cache.groups)


def test_storage_per_run(models, cpu_backend):
    e = _engine(models, "A")
    kv, st = e.model.storage_requests()
    extra = e.model.extra_storage_requests()
    # five runs; keys of two maps and values of another size in a store each, latents with their
    # rotated part in stores of one plane; runs that share tensors keep a store each
    assert sorted(kv) == [0, 1, 2, 3, 4] and st == {}
    assert kv[0] == kv[4] == KVRequest(2, 24, 9, planes=1)
    assert extra[(0, 0)] == extra[(4, 0)] == KVRequest(2, 20, 9, planes=1)
    assert kv[1] == kv[2] == KVRequest(1, 30, 0, planes=1)
    assert kv[3] == KVRequest(1, 48, 40, planes=1)
    assert e.cache.layer_kv(1).k.data_ptr() != e.cache.layer_kv(2).k.data_ptr()
    two = _engine(models, "B").model.storage_requests()[0]
    assert two[0] == KVRequest(2, 64, 100, planes=2) and two[2] == KVRequest(1, 128, 64, planes=2)
    assert two[1] == KVRequest(1, 80, 0, planes=1)


def test_a_window_gives_its_pages_back(models, cpu_backend):
    """400 tokens through B: the windowed stores keep two and three pages, the latents all of them."""
    _, cfg, P = models["B"]
    e = _engine(models, "B", cache_tokens=7 * 64, n_slots=1)
    toks = _tokens(320, 400, 9)
    s, at, outs = e.alloc_slot(), 0, []
    for size in (100, 28, 64, 128, 61):
        outs.append(e.step([(s, toks[at:at + size], list(range(size)))]))
        at += size
    outs += [e.step([(s, [t], [0])]) for t in toks[at:]]
    _close(torch.cat(outs), PB.logits(toks, P, cfg))
    assert sorted(len(g.pages_of(s)) for g in e.cache.groups) == [2, 3, 7, 7]
    e.free_slot(s)
    assert all(g.pool.n_free == g.pool.n_pages for g in e.cache.groups)


def test_greedy_generation_through_the_engines_loop(models, cpu_backend):
    _, cfg, P = models["A"]
    e = _engine(models, "A", cache_tokens=6 * 64, n_slots=3)
    prompts = [_tokens(211, n, 50 + n) for n in (5, 30, 1, 64)]
    out = e.generate(prompts, SamplingParams(max_new_tokens=8, temperature=0.0), max_batch=3)
    for p, got in zip(prompts, out):
        assert len(got) == 8
        ref = PB.logits(list(p) + got[:-1], P, cfg)[len(p) - 1:]
        for z, tok in zip(ref, got):      # only a near tie may differ
            assert float(z.max() - z[tok]) <= 1e-4 * float(z.abs().max())
    assert e.cache.slots.n_free == 3


def test_random_weights_mode_and_inspect(cpu_backend):
    for name in NAMES:
        cfg = BumulixConfig.from_json(BM.CONFIGS[name])
        e = Engine.random(cfg, seed=3, dtype="float32", device="cpu", cache_tokens=256)
        out = e.step([(e.alloc_slot(), [1, 2, 3], [2])])
        assert out.shape == (1, cfg.vocab_size) and torch.isfinite(out).all()
        assert e.model.n_params() >= cfg.n_params()       # fused products are filled up with zeros
    cfg = BumulixConfig.from_json(BM.CONFIGS["B"])        # where nothing is filled up
    e = Engine.random(cfg, seed=3, dtype="float32", device="cpu", cache_tokens=256)
    assert e.model.n_params() == cfg.n_params()
    info = e.inspect()
    assert info["architecture"] == "bumulix" and info["layers"] == 4 and info["tie_head"] is True
    small = Engine.random("bumulix-tiny", seed=1, dtype="float32", device="cpu", cache_tokens=256)
    assert small.step([(small.alloc_slot(), [5, 6], [1])]).shape[0] == 1


def test_command_line_and_trace_replay_take_the_design(cpu_backend, tmp_path, monkeypatch, capsys):
    import importlib.machinery
    import importlib.util
    from pathlib import Path

    import numpy as np
    from nimbus_infer_rs_b200.__main__ import main as cli
    folder = tmp_path / "m"
    assert cli(["random", "--preset", "bumulix-tiny", "--out", str(folder), "--seed", "5"]) == 0
    assert json.loads((folder / "config.json").read_text())["architecture"] == "Bumulix"
    capsys.readouterr()
    e = Engine.load(folder, dtype="float32", device="cpu", cache_tokens=128)
    want = e.step([(e.alloc_slot(), [3, 1, 4, 1, 5], [0, 4])])
    path = Path(__file__).resolve().parent.parent / "bin" / "trace_run"
    spec = importlib.util.spec_from_loader("trace_run_cli", importlib.machinery.SourceFileLoader(
        "trace_run_cli", str(path)))
    tr = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(tr)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [3, 1, 4], "want": [0]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [1, 5], "want": [1]}], "end": ["a"]}]
    monkeypatch.setattr("sys.stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    monkeypatch.setattr("sys.argv", ["trace_run", "--model", str(folder), "--dtype", "float32",
                                     "--out", str(tmp_path / "o"), "--max-tokens", "5", "--device", "cpu"])
    assert tr.main() == 0
    assert capsys.readouterr().out.split() == ["done", "0", "done", "1"]
    got = np.concatenate([np.fromfile(tmp_path / "o" / f"{i}.f32", dtype="<f4") for i in (0, 1)])
    _close(torch.from_numpy(got).view(2, -1), want)
