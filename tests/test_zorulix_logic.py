"""Zorulix without a GPU: its configuration and weight plan, and the engine's host side (stores of
keys and values of different sizes, layers that read another layer's store under a window of
their own, two mixers side by side, the recurrence's state and the convolution's inputs in one
row, slots, pages, batches, the generation loop) on the torch-CPU stand-in of the kernel library,
against the plain implementation."""
import copy
import io
import json

import pytest
import torch

import plain_zorulix as PZ
import zorulix_models as ZM
from nimbus_infer_rs_b200 import Engine, SamplingParams
from nimbus_infer_rs_b200.config import ConfigError, ZorulixConfig
from nimbus_infer_rs_b200.config.registry import load_config, resolve_architecture
from nimbus_infer_rs_b200.parts.base import KVRequest
from nimbus_infer_rs_b200.parts.masked_attention import MaskedAttention
from nimbus_infer_rs_b200.parts.routed_experts import RoutedExperts
from nimbus_infer_rs_b200.weights.loader import WeightError

NAMES = list(ZM.CONFIGS)


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("zorulix")
    return {n: ZM.make(root, n) for n in NAMES}


def _tokens(vocab, n, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def _close(got, ref, tol=3e-5):
    got, ref = got.double(), ref.double()
    assert got.shape == ref.shape
    assert float((got - ref).abs().max()) <= tol * float(ref.abs().max())


def _engine(models, name, **kw):
    kw.setdefault("cache_tokens", 1024)
    return Engine.load(models[name][0], dtype="float32", device="cpu", **kw)


def test_config_is_read_and_recognised(models, cpu_backend):
    arch, typed = load_config(models["A"][0])
    assert arch.name == "zorulix" and isinstance(typed, ZorulixConfig)
    assert resolve_architecture({"architecture": "zorulix"}).name == "zorulix"
    assert (typed.vocab_size, typed.width, typed.norm_eps, typed.embedding_scale, typed.side_dim) == \
        (211, 56, 3e-5, 5.0, 10)
    a = typed.layers[0].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.mask_size, a.kv_from) == (4, 2, 12, 20, 0.4, 9, None)
    assert (a.rot.dims, a.rot.base, a.rot.scaling()) == (12, 500.0, None)
    p = typed.layers[1].mixer
    assert p.left.rot.scaling() == {"factor": 4.0, "original": 64.0, "fast": 8.0, "slow": 0.5}
    r = p.right
    assert (r.heads, r.kv_heads, r.dim, r.vdim, r.taps, r.decay_rank) == (4, 2, 9, 13, 4, None)
    assert (p.left_scale, p.right_scale) == (1.4, 0.6)
    f = typed.layers[1].mlp
    assert (f.experts, f.top, f.ff, f.shared_ff) == (5, 3, 20, 28)
    assert typed.layers[2].mixer.kv_from == 0 and typed.layers[2].mlp is None
    assert typed.layers[3].mlp.shared_ff is None
    for n in NAMES:
        c = ZorulixConfig.from_json(ZM.CONFIGS[n])
        assert ZorulixConfig.from_json(c.to_json()) == c
    # the ranks come from the weight file and are carried by a config written here
    e = _engine(models, "A")
    r = e.config.layers[1].mixer.right
    assert (r.decay_rank, r.gate_rank) == ZM.RANKS["A"]
    assert ZorulixConfig.from_json(e.config.to_json()) == e.config
    # what is left out is absent, or follows from other sizes
    short = copy.deepcopy(ZM.CONFIGS["C"])
    for key in ("embedding",):
        del short[key]
    for key in ("kv_heads", "vdim", "scale"):
        del short["layers"][1]["mixer"]["left"][key]
    for key in ("left_scale", "right_scale"):
        del short["layers"][1]["mixer"][key]
    c = ZorulixConfig.from_json(short)
    m = c.layers[1].mixer
    assert (c.embedding_scale, c.side_dim, m.left_scale, m.right_scale) == (1.0, 0, 1.0, 1.0)
    assert (m.left.kv_heads, m.left.vdim, m.left.scale) == (m.left.heads, m.left.dim, m.left.dim ** -0.5)


def test_config_errors_name_every_bad_key():
    bad = copy.deepcopy(ZM.CONFIGS["A"])
    bad["layers"][0]["mixer"]["heads"] = 3                     # no multiple of kv_heads
    bad["layers"][0]["mlp"]["router"]["top"] = 9
    bad["layers"][1]["mixer"]["left"]["rot"]["dims"] = 12      # more than the head has
    del bad["layers"][1]["mixer"]["left"]["rot"]["scaling"]["fast"]
    bad["layers"][1]["mixer"]["left"]["kv_from"] = 0
    del bad["layers"][1]["mixer"]["right"]["conv"]
    bad["layers"][2]["mixer"]["kv_from"] = 2
    bad["layers"][3]["mlp"] = {"kind": "dense"}
    bad["layers"][4]["type"] = "windowed"
    bad["token_side"] = {"dim": 0}
    del bad["norm"]
    with pytest.raises(ConfigError) as e:
        ZorulixConfig.from_json(bad)
    msg = str(e.value)
    for piece in ("layers[0].mixer: heads", "top=9", "rot.dims", "scaling.fast", "left.kv_from", "right.conv",
                  "layers[2].mixer.kv_from", "dense", "windowed", "token_side.dim", "norm.eps"):
        assert piece in msg, piece
    for layer, change in ((2, {"kv_from": 1}), (4, {"kv_from": 2}), (2, {"vdim": 12}), (2, {"kv_heads": 1})):
        other = copy.deepcopy(ZM.CONFIGS["A"])
        other["layers"][layer]["mixer"].update(change)
        with pytest.raises(ConfigError, match="kv_from"):
            ZorulixConfig.from_json(other)


def test_weight_errors_are_listed_together(models, tmp_path):
    _, cfg, tensors = models["A"]
    t = dict(tensors)
    del t["l1.mix.right.k.conv"], t["l0.mlp.router.b"], t["l1.mix.left.o.b"]
    t["l0.mix.q.norm"] = torch.zeros(12)         # one head's instead of all heads'
    t["l2.mix.k"] = torch.zeros(24, 56)          # a reader has no keys of its own
    t["l2.norm2"] = torch.zeros(56)              # stands before a feed-forward that is not there
    folder = ZM.write_model(tmp_path / "bad", cfg, t)
    with pytest.raises(WeightError) as e:
        Engine.load(folder, dtype="float32", device="cpu")
    assert e.value.missing == ["l0.mlp.router.b", "l1.mix.left.o.b", "l1.mix.right.k.conv"]
    assert e.value.unexpected == ["l2.mix.k"]
    assert any("l0.mix.q.norm" in w for w in e.value.wrong_shape)


def test_parts_refuse_what_does_not_go_together():
    with pytest.raises(ValueError, match="qk_norm"):
        MaskedAttention(8, 1, 1, 8, 1.0, qk_norm="rows")
    with pytest.raises(ValueError, match="bias on the logits"):
        RoutedExperts(8, 4, 2, 8, scores="sigmoid", router_bias=True)


@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_and_token_by_token(models, cpu_backend, name):
    _, cfg, P = models[name]
    e = _engine(models, name)
    for n in (1, 2, 37, 80):
        toks = _tokens(cfg["vocab"], n, n)
        ref = PZ.logits(toks, P, cfg)
        s = e.alloc_slot()
        _close(e.step([(s, toks, list(range(n)))]), ref)
        e.free_slot(s)
        s = e.alloc_slot()
        _close(torch.cat([e.step([(s, [t], [0])]) for t in toks]), ref)
        e.free_slot(s)


@pytest.mark.parametrize("name", ["A", "D"])
def test_layer_by_layer(models, cpu_backend, name):
    _, cfg, P = models[name]
    e = _engine(models, name)
    snaps = []
    for l in e.model.layers:
        f = l.block.forward

        def tapped(ctx, x, layer, f=f):
            f(ctx, x, layer)
            snaps.append(x.clone())
        l.block.forward = tapped
    toks = _tokens(cfg["vocab"], 50, 5)
    e.step([(e.alloc_slot(), toks, [0])])
    ref = PZ.hidden_states(toks, P, cfg)
    assert len(snaps) == ref.shape[0] == len(cfg["layers"])
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
    _close(torch.cat(outs), PZ.logits(toks, P, cfg))


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
            _close(torch.stack(got[i]), PZ.logits(seqs[i], P, cfg)[heads[i] - 1:])
            e.free_slot(slots[i])
    assert all(g.pool.n_free == g.pool.n_pages for g in e.cache.groups)


def test_storage_of_owners_readers_and_pairs(models, cpu_backend):
    e = _engine(models, "A")
    kv, st = e.model.storage_requests()
    # readers keep nothing; the owner keeps what the longest window among them looks back at
    assert sorted(kv) == [0, 1, 3] and not e.model.extra_storage_requests()
    assert kv[0] == KVRequest(2, 12, 70, value_dim=20)
    assert kv[1] == KVRequest(1, 10, 33, value_dim=18) and kv[3] == KVRequest(2, 6, 5, value_dim=14)
    assert [e.model.kv_source(i) for i in range(5)] == [0, 1, 0, 3, 0]
    # a pair's state row: the recurrence's matrices and the convolution's last inputs
    def row(H, G, d, dv, taps):
        return -(-(H * d * dv + (taps - 1) * (2 * G * d + H * dv)) // 4) * 4
    assert {k: v.n_elements for k, v in st.items()} == {1: row(4, 2, 9, 13, 4), 3: row(3, 1, 6, 10, 2)}
    store = e.cache.layer_kv(0)
    assert store.k.shape[1:] == (2, 64, 12) and store.v.shape[1:] == (2, 64, 20)
    assert store.k.is_contiguous() and store.v.is_contiguous()
    a, b = store.k.data_ptr(), store.v.data_ptr()
    assert b == a + store.k.numel() * 4                # one plane behind the other
    # a reader that sees everything makes its owner keep everything
    assert _engine(models, "E").model.storage_requests()[0][0].window == 0
    assert _engine(models, "B").model.storage_requests()[0][0].window == 100


def test_a_window_gives_its_pages_back(models, cpu_backend):
    """400 tokens through B: every store keeps the pages its longest reader looks back at."""
    _, cfg, P = models["B"]
    e = _engine(models, "B", cache_tokens=7 * 64, n_slots=1)
    toks = _tokens(320, 400, 9)
    s, at, outs = e.alloc_slot(), 0, []
    for size in (100, 28, 64, 128, 61):
        outs.append(e.step([(s, toks[at:at + size], list(range(size)))]))
        at += size
    outs += [e.step([(s, [t], [0])]) for t in toks[at:]]
    _close(torch.cat(outs), PZ.logits(toks, P, cfg))
    assert sorted((g.request.window, len(g.pages_of(s))) for g in e.cache.groups) == [(64, 2), (100, 3), (128, 3)]
    e.free_slot(s)
    assert all(g.pool.n_free == g.pool.n_pages for g in e.cache.groups)


def test_greedy_generation_through_the_engines_loop(models, cpu_backend):
    _, cfg, P = models["A"]
    e = _engine(models, "A", cache_tokens=6 * 64, n_slots=3)
    prompts = [_tokens(211, n, 50 + n) for n in (5, 30, 1, 64)]
    out = e.generate(prompts, SamplingParams(max_new_tokens=8, temperature=0.0), max_batch=3)
    for p, got in zip(prompts, out):
        assert len(got) == 8
        ref = PZ.logits(list(p) + got[:-1], P, cfg)[len(p) - 1:]
        for z, tok in zip(ref, got):      # only a near tie may differ
            assert float(z.max() - z[tok]) <= 1e-4 * float(z.abs().max())
    assert e.cache.slots.n_free == 3


def test_random_weights_mode_and_inspect(cpu_backend):
    for name in NAMES:
        cfg = ZorulixConfig.from_json(ZM.CONFIGS[name])
        e = Engine.random(cfg, seed=3, dtype="float32", device="cpu", cache_tokens=256)
        out = e.step([(e.alloc_slot(), [1, 2, 3], [2])])
        assert out.shape == (1, cfg.vocab_size) and torch.isfinite(out).all()
        assert e.model.n_params() >= cfg.n_params()       # fused products are filled up with zeros
    # where nothing is filled up: sizes that are multiples of 8, one rank, eight heads and router rows
    full = ZM.model(64, 32, [
        ZM.one(ZM.attn(2, 1, 16, 16, 0.2, 9, 8), ZM.moe(16, 7, 2, 16)),
        ZM.two(ZM.attn(2, 1, 16, 24, 0.2, 9), {**ZM.delta(8, 8, 8, 8, 3), "decay_rank": 8, "gate_rank": 8},
               ZM.moe(8, 8, 3))], side=8)
    cfg = ZorulixConfig.from_json(full)
    e = Engine.random(cfg, seed=3, dtype="float32", device="cpu", cache_tokens=256)
    assert e.model.n_params() == cfg.n_params()
    info = e.inspect()
    assert info["architecture"] == "zorulix" and info["layers"] == 2 and info["tie_head"] is False
    small = Engine.random("zorulix-tiny", seed=1, dtype="float32", device="cpu", cache_tokens=256)
    assert small.step([(small.alloc_slot(), [5, 6], [1])]).shape[0] == 1


def test_command_line_and_trace_replay_take_the_design(cpu_backend, tmp_path, monkeypatch, capsys):
    import importlib.machinery
    import importlib.util
    from pathlib import Path

    import numpy as np
    from nimbus_infer_rs_b200.__main__ import main as cli
    folder = tmp_path / "m"
    assert cli(["random", "--preset", "zorulix-tiny", "--out", str(folder), "--seed", "5"]) == 0
    assert json.loads((folder / "config.json").read_text())["architecture"] == "Zorulix"
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
