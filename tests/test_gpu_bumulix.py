"""Bumulix on the GPU against the plain implementation, in 32-bit and in bfloat16: whole prompts,
token by token, portions, unequal batches, slots and pages used again, long decoding across
windows, greedy generation through the engine's own loop, configurations drawn at random, and a
test that changes mechanisms in the plain implementation and sees the comparison fail."""
import copy
import random

import pytest
import torch

import bumulix_models as BM
import plain_bumulix as PB
from gpu_helpers import DTYPES
from nimbus_infer_rs_b200 import Engine, SamplingParams

pytestmark = pytest.mark.gpu
NAMES = list(BM.CONFIGS)
# In 32-bit: largest |engine - plain| relative to the largest |plain logit|.  In bfloat16: a row's
# root-mean-square difference over the vocabulary relative to the spread of the logits (a head's
# difference of two maps is brought to unit size, so rounding of a small difference counts in
# full); the mechanisms alone are held to 2e-5 and 2e-2 in test_gpu_bumulix_kernels.py.
TOL = {"float32": 1e-4, "bfloat16": 6e-2}


def assert_close(got, ref, dtype, what=""):
    """In 32-bit every row within the tolerance.  In bfloat16 one row in fifty (at least one) may
    be over it, none over twice it."""
    got, ref = got.detach().double().cpu(), ref.detach().double().cpu()
    assert got.shape == ref.shape, f"{what}: shape {tuple(got.shape)} vs {tuple(ref.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite values"
    err = (got - ref).reshape(got.shape[0], -1)
    rows = err.abs().max(1).values / float(ref.abs().max()) if dtype == "float32" \
        else err.square().mean(1).sqrt() / float(ref.square().mean().sqrt())
    over = int((rows > TOL[dtype]).sum())
    allowed = 0 if dtype == "float32" else max(1, got.shape[0] // 50)
    assert over <= allowed and float(rows.max()) <= 2 * TOL[dtype], \
        f"{what}: {over} rows over {TOL[dtype]:.0e} (allowed {allowed}), worst {float(rows.max()):.3e} " \
        f"at row {int(rows.argmax())}"


def _cases(names):
    """Every configuration in both precisions, except C in bfloat16: its norms over one or two
    numbers are sign functions, which rounding flips."""
    return [(n, d) for n in names for d in DTYPES if not (n == "C" and d == "bfloat16")]


@pytest.fixture(scope="module", autouse=True)
def _few_threads():
    """The plain implementation's matrices are small: many threads only wait for one another."""
    n = torch.get_num_threads()
    torch.set_num_threads(2)
    yield
    torch.set_num_threads(n)


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("bumulix")
    return {n: BM.make(root, n) for n in NAMES}


def _tokens(vocab, n, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def _engine(models, name, dtype, cache_tokens=1024, **kw):
    return Engine.load(models[name][0], dtype=dtype, cache_tokens=cache_tokens, **kw)


@pytest.mark.parametrize("name,dtype", _cases(NAMES))
def test_each_request_alone_and_whole(models, name, dtype):
    _, cfg, P = models[name]
    e = _engine(models, name, dtype)
    for i, n in enumerate((1, 2, 33, 64, 65, 190)):
        toks = _tokens(cfg["vocab"], n, 10 + i)
        s = e.alloc_slot()
        out = e.step([(s, toks, list(range(n)))])
        e.free_slot(s)
        assert_close(out, PB.logits(toks, P, cfg), dtype, f"{name} whole, {n} tokens")
    e.check_errors()


@pytest.mark.parametrize("name", ["A", "E"])
def test_layer_by_layer_in_32_bit(models, name):
    _, cfg, P = models[name]
    e = _engine(models, name, "float32")
    e.step_graphs = None
    snaps, S = [], cfg.get("streams", 1)
    for l in e.model.layers:
        f = l.block.forward

        def tapped(ctx, x, layer, f=f):
            f(ctx, x, layer)
            snaps.append((x.view(x.shape[0], S, -1).sum(1) if ctx.streams_sum is None
                          else ctx.streams_sum).clone())
        l.block.forward = tapped
    toks = _tokens(cfg["vocab"], 90, 5)
    e.step([(e.alloc_slot(), toks, [0])])
    ref = PB.hidden_states(toks, P, cfg)
    assert len(snaps) == ref.shape[0] == len(cfg["layers"])
    for i, (got, want) in enumerate(zip(snaps, ref)):
        assert_close(got[:90], want, "float32", f"stream after layer run {i}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B"])
def test_recorded_steps_give_what_plain_launches_give(models, name, dtype):
    """A step whose shape comes again is replayed from a CUDA graph: bit for bit the same."""
    _, cfg, _ = models[name]
    e, plainly = _engine(models, name, dtype), _engine(models, name, dtype)
    plainly.step_graphs = None
    for n in (1, 70, 1, 70, 1, 70):
        toks = _tokens(cfg["vocab"], n, n)
        s, t = e.alloc_slot(), plainly.alloc_slot()
        a, b = e.step([(s, toks, list(range(n)))]), plainly.step([(t, toks, list(range(n)))])
        for k in range(3):
            a = torch.cat([a, e.step([(s, [k + 1], [0])])])
            b = torch.cat([b, plainly.step([(t, [k + 1], [0])])])
        e.free_slot(s)
        plainly.free_slot(t)
        assert torch.equal(a, b)
    assert e.step_graphs.replays > 0


@pytest.mark.parametrize("name,dtype", _cases(NAMES))
def test_last_tokens_one_by_one(models, name, dtype):
    _, cfg, P = models[name]
    e = _engine(models, name, dtype)
    for n, head in ((34, 1), (190, 140)):
        toks = _tokens(cfg["vocab"], n, n)
        s = e.alloc_slot()
        outs = [e.step([(s, toks[:head], [head - 1])])]
        for t in range(head, n):
            outs.append(e.step([(s, [toks[t]], [0])]))
        e.free_slot(s)
        assert_close(torch.cat(outs), PB.logits(toks, P, cfg)[head - 1:], dtype, f"{name} from {head} of {n}")


@pytest.mark.parametrize("name,dtype", _cases(["A", "B", "D", "E"]))
def test_portions_of_several_sizes(models, name, dtype):
    """Portions that start inside a window and end on and beside page ends, down to one token."""
    _, cfg, P = models[name]
    e = _engine(models, name, dtype)
    toks = _tokens(cfg["vocab"], 203, 3)
    s, at, outs = e.alloc_slot(), 0, []
    for size in (2, 61, 1, 2, 64, 3, 70):
        outs.append(e.step([(s, toks[at:at + size], list(range(size)))]))
        at += size
    assert_close(torch.cat(outs), PB.logits(toks, P, cfg), dtype, f"{name} portions")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B"])
def test_unequal_batches_on_slots_and_pages_used_again(models, name, dtype):
    """Batches of unequal prompts, decoded together while the shorter ones end; the cache holds
    one batch, so the next one gets the same slots and pages."""
    _, cfg, P = models[name]
    e = _engine(models, name, dtype, cache_tokens=6 * 64, n_slots=3)
    V = cfg["vocab"]
    for turn, lens in enumerate(((130, 7, 66), (64, 129, 2), (1, 1, 190))):
        seqs = [_tokens(V, n, 31 * turn + i) for i, n in enumerate(lens)]
        heads = [max(1, n - 3 - 2 * i) for i, n in enumerate(lens)]
        slots = [e.alloc_slot() for _ in lens]
        got = {i: [] for i in range(3)}
        out = e.step([(slots[i], t[:h], [0, h - 1]) for i, (t, h) in enumerate(zip(seqs, heads))])
        for i in range(3):
            got[i] += [out[2 * i], out[2 * i + 1]]
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
            ref = PB.logits(seqs[i], P, cfg)
            places = [0, heads[i] - 1] + list(range(heads[i], lens[i]))
            assert_close(torch.stack(got[i]), ref[places], dtype, f"{name} batch {turn} request {i}")
            e.free_slot(slots[i])
    assert all(g.pool.n_free == g.pool.n_pages for g in e.cache.groups)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["B", "D"])
def test_long_decoding_from_the_first_token(models, name, dtype):
    """Windows pass over decoded tokens; pages behind them are given back."""
    _, cfg, P = models[name]
    e = _engine(models, name, dtype)
    toks = _tokens(cfg["vocab"], 250, 9)
    s = e.alloc_slot()
    outs = [e.step([(s, [t], [0])]) for t in toks]
    assert_close(torch.cat(outs), PB.logits(toks, P, cfg), dtype, "250 tokens one by one")


def test_greedy_generation_through_the_engines_loop(models):
    _, cfg, P = models["B"]
    e = _engine(models, "B", "float32", cache_tokens=8 * 64, n_slots=3)
    prompts = [_tokens(320, n, 70 + n) for n in (5, 63, 1, 120)]
    out = e.generate(prompts, SamplingParams(max_new_tokens=12, temperature=0.0), max_batch=3)
    for p, got in zip(prompts, out):
        assert len(got) == 12
        ref = PB.logits(list(p) + got[:-1], P, cfg)[len(p) - 1:]
        for z, tok in zip(ref, got):      # only a near tie may differ
            assert float(z.max() - z[tok]) <= 2 * TOL["float32"] * float(z.abs().max())
    assert e.cache.slots.n_free == 3


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_decode_session_is_recorded_and_a_row_may_stop_early(models, dtype):
    """Generation runs in a recorded decode session; a sequence that meets a stop token becomes a
    padding row of it, and the others go on exactly as they do without the stop."""
    e = _engine(models, "B", dtype, cache_tokens=8 * 64)
    assert e.graph_safe
    prompts = [_tokens(320, n, 7 + n) for n in (12, 70, 3)]
    free = e.generate(prompts, SamplingParams(max_new_tokens=16, temperature=0.0))
    assert free == e.generate(prompts, SamplingParams(max_new_tokens=16, temperature=0.0))
    stop = free[0][4]
    out = e.generate(prompts, SamplingParams(max_new_tokens=16, temperature=0.0, stop_tokens=[stop]))
    assert len(out[0]) <= 5
    for f, o in zip(free, out):
        cut = f.index(stop) + 1 if stop in f else len(f)
        assert o == f[:cut]
    assert e.cache.slots.n_free == e.cache.n_slots


def test_the_comparison_sees_a_changed_mechanism(models):
    """The tests above would not notice a mechanism that changes nothing: change each in the
    plain implementation and see the engine's logits move away by far more than the tolerance."""
    _, cfg, P = models["A"]
    e = _engine(models, "A", "float32")
    toks = _tokens(211, 60, 2)
    s = e.alloc_slot()
    out = e.step([(s, toks, list(range(60)))]).double().cpu()
    e.free_slot(s)

    def moved(Pmod=None, cfgmod=None):
        ref = PB.logits(toks, Pmod or P, cfgmod or cfg)
        return float((out - ref).abs().max()) / float(ref.abs().max())

    assert moved() <= TOL["float32"]

    def each(kind, f):
        return lambda c: [f(l["mixer"]) for l in c["layers"] if l["type"] == kind]

    pairs, latents = (lambda f: each("attention", f)), (lambda f: each("latent_attention", f))
    for n, change in enumerate((
            pairs(lambda m: m.update(diff=m["diff"] + 0.05)),
            pairs(lambda m: m.update(scale=m["scale"] * 1.05)),
            pairs(lambda m: m["mask"].update(size=m["mask"]["size"] + 1)),
            pairs(lambda m: m["mask"].update(size=m["mask"]["size"] - 1)),
            pairs(lambda m: m.pop("mask", None)),
            latents(lambda m: m.update(scale=0.31)),
            latents(lambda m: m["rot"].update(base=520.0)),
            latents(lambda m: m["rot"].update(dims=4)),
            latents(lambda m: m["rot"].pop("scaling", None)),
            latents(lambda m: m["rot"]["scaling"].update(factor=4.5)),
            latents(lambda m: m["rot"]["scaling"].update(original=32)),
            lambda c: c.update(residual_mult=0.72),
            lambda c: c.update(logit_softcap=12.5),
            lambda c: c.pop("logit_softcap"),
            lambda c: c.update(norm={"eps": 1e-2}))):
        other = copy.deepcopy(cfg)
        change(other)
        assert moved(None, other) > 1e-3, n
    for name in ("l0.hc1.in", "l0.hc1.out", "l0.hc1.mix", "l1.hc2.in", "l1.hc2.out", "l1.hc2.mix", "l0.ls1",
                 "l1.ls2", "l0.norm1", "l1.norm2", "l0.mix.lq1", "l0.mix.lk2", "l1.mix.dq.norm",
                 "l1.mix.dkv.norm", "l1.mix.g", "l1.mix.uk", "l1.mix.uv", "l3.mix.v", "final.norm"):
        other = dict(P)
        other[name] = P[name] * 0.7 + 0.2
        assert moved(other) > 1e-3, name
    mixed = {k: (v.T.contiguous() if k.endswith(".mix") and "hc" in k else v) for k, v in P.items()}
    assert moved(mixed) > 1e-3                       # from and to exchanged


def test_trace_replay_as_a_program(models, tmp_path):
    """bin/trace_run as a subprocess on a Bumulix folder: three requests of unequal lengths in one
    batch, decoded together while the shorter ones end, with exactly the tokens they hold as
    --max-tokens."""
    import json
    import subprocess
    from pathlib import Path

    import numpy as np
    folder, cfg, P = models["D"]
    root = Path(__file__).resolve().parent.parent
    V = cfg["vocab"]
    seqs = {"a": _tokens(V, 150, 1), "b": _tokens(V, 70, 2), "c": _tokens(V, 9, 3)}
    heads = {"a": 140, "b": 66, "c": 1}
    steps = [{"step": 0, "entries": [{"id": k, "tokens": seqs[k][:heads[k]], "want": [heads[k] - 1]}
                                     for k in "abc"], "end": []}]
    k = 0
    while True:
        live = [r for r in "abc" if heads[r] + k < len(seqs[r])]
        if not live:
            break
        steps.append({"step": len(steps), "entries": [{"id": r, "tokens": [seqs[r][heads[r] + k]], "want": [0]}
                                                      for r in live],
                      "end": [r for r in live if heads[r] + k + 1 == len(seqs[r])]})
        k += 1
    out = tmp_path / "out"
    proc = subprocess.Popen([str(root / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32",
                             "--out", str(out), "--max-tokens", str(sum(len(v) for v in seqs.values()))],
                            stdin=subprocess.PIPE, stdout=subprocess.PIPE, text=True, cwd="/")
    for st in steps:
        proc.stdin.write(json.dumps(st) + "\n")
        proc.stdin.flush()
        assert proc.stdout.readline().strip() == f"done {st['step']}"
    proc.stdin.close()
    assert proc.wait(timeout=120) == 0
    refs = {r: PB.logits(seqs[r], P, cfg) for r in "abc"}
    for st in steps:
        got = torch.from_numpy(np.fromfile(out / f"{st['step']}.f32", dtype="<f4").reshape(-1, V))
        want = [refs[e["id"]][heads[e["id"]] - 1 + st["step"]] for e in st["entries"]]
        assert_close(got, torch.stack(want), "float32", f"step {st['step']}")


# ----------------------------------------------------------------------------- drawn at random
def random_config(rng):
    def a_pair():
        d = rng.choice([8, 16, 32, 40, 64, 24, 20])
        dv = 2 * d if rng.random() < 0.65 else rng.choice([16, 32, 64, 72, 128, 30])
        G = rng.choice([1, 2, 3])
        return BM.pair(G * rng.choice([1, 2, 3, 4, 5]), G, d, dv, rng.choice([d ** -0.5, 0.1, 0.2]),
                       rng.choice([0.2, 0.5, 0.8]),
                       rng.choice([None, 1, 7, 63, 64, 65, 90, 100, 128, 130, 200]))

    def a_latent():
        r = rng.choice([2, 8, 16, 32, 64, 10, 80])
        scaling = None if rng.random() < 0.3 else \
            rng.choice([(2.0, 32, 4.0, 0.5), (8.0, 128, 32.0, 1.0), (40.0, 4096, 32.0, 1.0)])
        return BM.latent(rng.choice([1, 2, 3, 5, 8]), rng.choice([16, 24, 64, 30]), r,
                         rng.choice([16, 32, 72, 20]), rng.choice([32, 64, 80, 128, 200, 36]),
                         rng.choice([16, 40, 96, 50]), rng.choice([0.08, 0.15, 0.2]),
                         rng.choice([100.0, 10000.0, 500000.0]), scaling)

    layers = []
    for _ in range(rng.randint(2, 6)):
        if layers and rng.random() < 0.25:            # a layer on an earlier layer's tensors
            j = rng.randrange(len(layers))
            while layers[j].get("weights_of") is not None:
                j = layers[j]["weights_of"]
            layers.append({**layers[j], "weights_of": j})
        else:
            layers.append(BM.layer(rng.choice([a_pair, a_latent])(), rng.choice([None, 40, 64, 256, 100])))
    return BM.model(rng.choice([97, 300, 1000, 450]), rng.choice([64, 100, 128, 96, 328]), layers,
                    streams=rng.choice([1, 2, 3, 4, 4, 6]), mult=rng.choice([0.3, 0.5, 1.0]),
                    cap=rng.choice([15.0, 30.0, 50.0]), eps=rng.choice([1e-5, 1e-6]))


@pytest.mark.parametrize("seed", range(12))
def test_a_random_configuration(tmp_path, seed):
    """Three unequal requests in one batch, prompts with every logit wanted, then decoded together
    while the shorter ones end, in both precisions."""
    rng = random.Random(seed)
    cfg = random_config(rng)
    P = BM.make_tensors(cfg, seed)
    folder = BM.write_model(tmp_path / "m", cfg, P)
    lens = [rng.choice([300, 140, 70]), rng.choice([1, 9, 66]), rng.choice([130, 200])]
    heads = [max(1, n - rng.choice([3, 20, 40])) for n in lens]
    seqs = [_tokens(cfg["vocab"], n, 100 * seed + i) for i, n in enumerate(lens)]
    refs = [PB.logits(t, P, cfg) for t in seqs]
    for dtype in DTYPES:
        e = Engine.load(folder, dtype=dtype, cache_tokens=1024)
        slots = [e.alloc_slot() for _ in lens]
        out = e.step([(slots[i], seqs[i][:heads[i]], list(range(heads[i]))) for i in range(3)])
        got = {i: [g] for i, g in enumerate(torch.split(out, heads))}
        k = 0
        while True:
            live = [i for i in range(3) if heads[i] + k < lens[i]]
            if not live:
                break
            out = e.step([(slots[i], [seqs[i][heads[i] + k]], [0]) for i in live])
            for j, i in enumerate(live):
                got[i].append(out[j:j + 1])
            k += 1
        e.check_errors()
        for i in range(3):
            assert_close(torch.cat(got[i]), refs[i], dtype, f"request {i}; {cfg}")
