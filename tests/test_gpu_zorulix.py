"""Zorulix on the GPU against the plain implementation, in 32-bit and in bfloat16: whole prompts,
token by token, portions, unequal batches, slots and pages used again, long decoding across
windows, greedy generation through the engine's own loop, configurations drawn at random, and a
test that changes mechanisms in the plain implementation and sees the comparison fail."""
import copy
import random

import pytest
import torch

import plain_zorulix as PZ
import zorulix_models as ZM
from gpu_helpers import DTYPES
from nimbus_infer_rs_b200 import Engine, SamplingParams

pytestmark = pytest.mark.gpu
NAMES = list(ZM.CONFIGS)
# In 32-bit: largest |engine - plain| relative to the largest |plain logit|.  In bfloat16: a row's
# root-mean-square difference over the vocabulary relative to the spread of the logits; the
# mechanisms alone are held to tighter figures in test_gpu_zorulix_kernels.py.
TOL = {"float32": 1e-4, "bfloat16": 6e-2}
# A router's choice between experts whose logits are closer than this is a close call that
# rounding may settle either way; the plain implementation then follows the engine (and insists on
# its own choice everywhere else).
MARGIN = {"float32": 1e-3, "bfloat16": 0.25}


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
    """Every configuration in both precisions, except C in bfloat16: unit vectors of one number are
    sign functions, which rounding flips."""
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
    root = tmp_path_factory.mktemp("zorulix")
    return {n: ZM.make(root, n) for n in NAMES}


def _tokens(vocab, n, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


class Routed:
    """Notes what the router kernel chose, per slot, at every position of every layer with routed
    experts, for the steps that go through ``Engine.step``."""

    def __init__(self, engine):
        self.by_slot, self._calls = {}, []
        ops, orig, step, alloc = engine.ops, engine.ops.moe_route, engine.step, engine.alloc_slot

        def tapped(logits, col, n_experts, top, renormalize, layout, idx, weight, *bias):
            orig(logits, col, n_experts, top, renormalize, layout, idx, weight, *bias)
            self._calls.append(idx.clone())

        def stepped(entries):
            ops.moe_route = tapped
            try:
                out = step(entries)
            finally:
                del ops.moe_route                    # the class's method is back
            calls, self._calls = [c.cpu().long() for c in self._calls], []
            at = 0
            for e in entries:
                n = len(e[1])
                mine = [c[at:at + n] for c in calls]
                old = self.by_slot.get(e[0])
                self.by_slot[e[0]] = mine if old is None else [torch.cat([a, b]) for a, b in zip(old, mine)]
                at += n
            return out

        def allocated():
            slot = alloc()
            self.by_slot.pop(slot, None)
            return slot

        engine.step, engine.alloc_slot = stepped, allocated


def _engine(folder, dtype, cache_tokens=1024, tap=True, **kw):
    e = Engine.load(folder, dtype=dtype, cache_tokens=cache_tokens, **kw)
    if tap:
        e.step_graphs = None               # every launch goes through Python: the tap sees it
        e.routed = Routed(e)
    return e


def _plain(e, slot, toks, P, cfg, dtype):
    """The plain logits, with the engine's choice of experts where it is a close call."""
    layers = [i for i, l in enumerate(cfg["layers"]) if l["mlp"]]

    def choices(i, z):
        idx = e.routed.by_slot[slot][layers.index(i)]
        assert idx.shape[0] == z.shape[0]
        taken = torch.zeros_like(z, dtype=torch.bool).scatter(1, idx, True)
        worst = z.masked_fill(~taken, float("inf")).min(1).values
        best = z.masked_fill(taken, float("-inf")).max(1).values
        assert taken.sum(1).eq(idx.shape[1]).all()
        assert float((best - worst).max()) <= MARGIN[dtype], "an expert far from the best was chosen"
        return idx
    return PZ.logits(toks, P, cfg, choices=choices)


@pytest.mark.parametrize("name,dtype", _cases(NAMES))
def test_each_request_alone_and_whole(models, name, dtype):
    folder, cfg, P = models[name]
    e = _engine(folder, dtype)
    for i, n in enumerate((1, 2, 33, 64, 65, 190)):
        toks = _tokens(cfg["vocab"], n, 10 + i)
        s = e.alloc_slot()
        out = e.step([(s, toks, list(range(n)))])
        e.free_slot(s)
        assert_close(out, _plain(e, s, toks, P, cfg, dtype), dtype, f"{name} whole, {n} tokens")
    e.check_errors()


@pytest.mark.parametrize("name", ["A", "B", "E"])
def test_layer_by_layer_in_32_bit(models, name):
    folder, cfg, P = models[name]
    e = _engine(folder, "float32", tap=False)
    e.step_graphs = None
    snaps = []
    for l in e.model.layers:
        f = l.block.forward

        def tapped(ctx, x, layer, f=f):
            f(ctx, x, layer)
            snaps.append(x.clone())
        l.block.forward = tapped
    toks = _tokens(cfg["vocab"], 90, 5)
    e.step([(e.alloc_slot(), toks, [0])])
    ref = PZ.hidden_states(toks, P, cfg)
    assert len(snaps) == ref.shape[0] == len(cfg["layers"])
    for i, (got, want) in enumerate(zip(snaps, ref)):
        assert_close(got[:90], want, "float32", f"stream after layer {i}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B"])
def test_recorded_steps_give_what_plain_launches_give(models, name, dtype):
    """A step whose shape comes again is replayed from a CUDA graph: bit for bit the same."""
    folder, cfg, _ = models[name]
    e, plainly = _engine(folder, dtype, tap=False), _engine(folder, dtype, tap=False)
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
    folder, cfg, P = models[name]
    e = _engine(folder, dtype)
    for n, head in ((34, 1), (190, 140)):
        toks = _tokens(cfg["vocab"], n, n)
        s = e.alloc_slot()
        outs = [e.step([(s, toks[:head], [head - 1])])]
        for t in range(head, n):
            outs.append(e.step([(s, [toks[t]], [0])]))
        e.free_slot(s)
        assert_close(torch.cat(outs), _plain(e, s, toks, P, cfg, dtype)[head - 1:], dtype,
                     f"{name} from {head} of {n}")


@pytest.mark.parametrize("name,dtype", _cases(["A", "B", "D", "E"]))
def test_portions_of_several_sizes(models, name, dtype):
    """Portions that start inside a window and end on and beside page ends, down to one token."""
    folder, cfg, P = models[name]
    e = _engine(folder, dtype)
    toks = _tokens(cfg["vocab"], 203, 3)
    s, at, outs = e.alloc_slot(), 0, []
    for size in (2, 61, 1, 2, 64, 3, 70):
        outs.append(e.step([(s, toks[at:at + size], list(range(size)))]))
        at += size
    assert_close(torch.cat(outs), _plain(e, s, toks, P, cfg, dtype), dtype, f"{name} portions")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "E"])
def test_unequal_batches_on_slots_and_pages_used_again(models, name, dtype):
    """Batches of unequal prompts, decoded together while the shorter ones end; the cache holds
    one batch, so the next one gets the same slots and pages."""
    folder, cfg, P = models[name]
    e = _engine(folder, dtype, cache_tokens=6 * 64, n_slots=3)
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
            ref = _plain(e, slots[i], seqs[i], P, cfg, dtype)
            places = [0, heads[i] - 1] + list(range(heads[i], lens[i]))
            assert_close(torch.stack(got[i]), ref[places], dtype, f"{name} batch {turn} request {i}")
            e.free_slot(slots[i])
    assert all(g.pool.n_free == g.pool.n_pages for g in e.cache.groups)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_request_is_what_it_is_alone(models, dtype):
    """The same request alone and as one of a mixed batch (prompts, portions and single tokens in
    one step), on other slots and pages: equal within rounding, whatever stands beside it."""
    folder, cfg, P = models["B"]
    alone, mixed = _engine(folder, dtype), _engine(folder, dtype)
    toks, other = _tokens(320, 150, 1), _tokens(320, 180, 2)
    s = alone.alloc_slot()
    a = torch.cat([alone.step([(s, toks[:100], list(range(100)))])] +
                  [alone.step([(s, [t], [0])]) for t in toks[100:]])
    ref = _plain(alone, s, toks, P, cfg, dtype)
    o, s = mixed.alloc_slot(), mixed.alloc_slot()
    outs, at, oat = [], 0, 0
    for n, on in ((3, 64), (60, 1), (1, 30), (36, 2), *[(1, 1 + i % 2) for i in range(50)]):
        want = list(range(n))
        out = mixed.step([(o, other[oat:oat + on], [0]), (s, toks[at:at + n], want)])
        outs.append(out[1:])
        at += n
        oat += on
    assert_close(a, ref, dtype, "alone")
    assert_close(torch.cat(outs), _plain(mixed, s, toks, P, cfg, dtype), dtype, "in a mixed batch")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["B", "D"])
def test_long_decoding_from_the_first_token(models, name, dtype):
    """Windows pass over decoded tokens; pages behind them are given back."""
    folder, cfg, P = models[name]
    e = _engine(folder, dtype)
    toks = _tokens(cfg["vocab"], 250, 9)
    s = e.alloc_slot()
    outs = [e.step([(s, [t], [0])]) for t in toks]
    assert_close(torch.cat(outs), _plain(e, s, toks, P, cfg, dtype), dtype, "250 tokens one by one")


def test_greedy_generation_through_the_engines_loop(models):
    folder, cfg, P = models["B"]
    e = _engine(folder, "float32", cache_tokens=8 * 64, n_slots=3, tap=False)
    prompts = [_tokens(320, n, 70 + n) for n in (5, 63, 1, 120)]
    out = e.generate(prompts, SamplingParams(max_new_tokens=12, temperature=0.0), max_batch=3)
    for p, got in zip(prompts, out):
        assert len(got) == 12
        ref = PZ.logits(list(p) + got[:-1], P, cfg)[len(p) - 1:]
        for z, tok in zip(ref, got):      # only a near tie may differ
            assert float(z.max() - z[tok]) <= 2 * TOL["float32"] * float(z.abs().max())
    assert e.cache.slots.n_free == 3


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_decode_session_is_recorded_and_a_row_may_stop_early(models, dtype):
    """Generation runs in a recorded decode session; a sequence that meets a stop token becomes a
    padding row of it, and the others go on exactly as they do without the stop."""
    e = _engine(models["B"][0], dtype, cache_tokens=8 * 64, tap=False)
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
    folder, cfg, P = models["A"]
    e = _engine(folder, "float32", tap=False)
    toks = _tokens(211, 60, 2)
    s = e.alloc_slot()
    out = e.step([(s, toks, list(range(60)))]).double().cpu()
    e.free_slot(s)

    def moved(Pmod=None, cfgmod=None):
        ref = PZ.logits(toks, Pmod or P, cfgmod or cfg)
        return float((out - ref).abs().max()) / float(ref.abs().max())

    assert moved() <= TOL["float32"]
    for n, change in enumerate((
            lambda c: c[0]["mixer"].update(scale=0.43),
            lambda c: c[0]["mixer"]["mask"].update(size=10),
            lambda c: c[0]["mixer"]["mask"].update(size=8),
            lambda c: c[0]["mixer"]["rot"].update(base=520.0),
            lambda c: c[0]["mixer"]["rot"].update(dims=10),
            lambda c: c[2]["mixer"]["mask"].update(size=30),
            lambda c: c[2]["mixer"]["rot"].update(dims=8),
            lambda c: c[4]["mixer"]["mask"].update(size=5),
            lambda c: c[4]["mixer"].update(scale=0.53),
            lambda c: c[1]["mixer"].update(left_scale=1.45),
            lambda c: c[1]["mixer"].update(right_scale=0.65),
            lambda c: c[3]["mixer"].update(left_scale=-0.75),
            lambda c: c[1]["mixer"]["left"].update(scale=0.53),
            lambda c: c[1]["mixer"]["left"]["mask"].update(size=32),
            lambda c: c[1]["mixer"]["left"]["rot"].pop("scaling"),
            lambda c: c[1]["mixer"]["left"]["rot"]["scaling"].update(factor=4.5),
            lambda c: c[1]["mixer"]["left"]["rot"]["scaling"].update(original=32),
            lambda c: c[1]["mixer"]["left"]["rot"]["scaling"].update(fast=1.0),
            lambda c: c[0]["mlp"]["router"].update(top=1),
            lambda c: c[1]["mlp"]["router"].update(top=2),
            lambda c: c[1]["mlp"].pop("shared"))):
        other = copy.deepcopy(cfg)
        change(other["layers"])
        assert moved(None, other) > 1e-3, n
    for change in (dict(embedding={"scale": 5.1}), dict(norm={"eps": 1e-2})):
        assert moved(None, {**cfg, **change}) > 1e-3, change
    R = "l1.mix.right."
    for name in ("l0.norm1", "l1.norm2", "l0.mix.q.b", "l0.mix.k.b", "l0.mix.v.b", "l0.mix.q.norm",
                 "l0.mix.k.norm", "l2.mix.q.norm", "l2.mix.q.b", "l1.mix.left.q.b", "l1.mix.left.k.b",
                 "l1.mix.left.v.b", "l1.mix.left.o.b", R + "q", R + "k", R + "v", R + "q.conv", R + "k.conv",
                 R + "v.conv", R + "b", R + "a1", R + "a2", R + "A_log", R + "dt_bias", R + "g1", R + "g2",
                 R + "norm", R + "o", "l0.mlp.router.b", "l1.mlp.shared.up",
                 "l1.mlp.shared.sg", "side.embed", "l2.side.gate", "l3.side.proj", "l4.side.norm", "final.norm"):
        other = dict(P)
        other[name] = P[name] * 0.7 + 0.2
        assert moved(other) > 1e-3, name

    for name in ("l0.mlp.e{}.gate", "l1.mlp.e{}.up", "l4.mlp.e{}.down"):       # of every expert
        assert moved({k: v * 0.7 + 0.2 if any(k == name.format(e) for e in range(7)) else v
                      for k, v in P.items()}) > 1e-3, name

    def swapped(name, value):
        orig = getattr(PZ, name)
        setattr(PZ, name, value)
        try:
            return moved()
        finally:
            setattr(PZ, name, orig)
    attend, sigmoid_walk = PZ.attend, PZ.delta_walk
    assert swapped("attend", lambda q, k, v, see, scale, sink: attend(q, k, v, see, scale, False)) > 1e-3
    assert swapped("unit_vectors", lambda x: x) > 1e-3
    assert swapped("over_rms", lambda x, eps: x / torch.sqrt((x * x).mean(-1, keepdim=True) + 100 * eps)) > 1e-4
    assert swapped("delta_walk", lambda q, k, v, g, b: sigmoid_walk(q, k, v, torch.ones_like(g), b)) > 1e-3
    assert swapped("delta_walk", lambda q, k, v, g, b: sigmoid_walk(q, k, v, g, torch.ones_like(b))) > 1e-3
    assert swapped("causal_conv", lambda x, w: x * w[:, -1]) > 1e-3


def test_trace_replay_as_a_program(models, tmp_path):
    """bin/trace_run as a subprocess on a Zorulix folder: three requests of unequal lengths in one
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
    refs = {r: PZ.logits(seqs[r], P, cfg) for r in "abc"}
    for st in steps:
        got = torch.from_numpy(np.fromfile(out / f"{st['step']}.f32", dtype="<f4").reshape(-1, V))
        want = [refs[e["id"]][heads[e["id"]] - 1 + st["step"]] for e in st["entries"]]
        assert_close(got, torch.stack(want), "float32", f"step {st['step']}")


# ----------------------------------------------------------------------------- drawn at random
def random_config(rng):
    WINDOWS = [None, 1, 7, 63, 64, 65, 90, 100, 128, 130, 200]

    def sizes():
        d = rng.choice([8, 16, 32, 40, 48, 64, 96, 128, 20])
        return d, rng.choice([d, d, 2 * d if d <= 64 else d, 16, 32, 64, 128, 24, 30])

    def rotation(d):
        dims = rng.choice([d, d, d // 2 // 2 * 2])
        return {"rot": dims, "base": rng.choice([100.0, 10000.0, 500000.0])} if dims else {}

    def attention(heads_over=None):
        d, dv = sizes()
        G = rng.choice([1, 2, 3])
        return ZM.attn(G * rng.choice([1, 2, 3, 4, 8]), G, d, dv, rng.choice([d ** -0.5, 0.1, 0.2]),
                       rng.choice(WINDOWS), **rotation(d))

    def pair():
        left = attention()
        if left.get("rot") and rng.random() < 0.7:
            left["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), rng.choice(
                [(2.0, 32, 4.0, 0.5), (8.0, 128, 32.0, 1.0), (40.0, 4096, 32.0, 1.0)])))
        G = rng.choice([1, 2, 4])
        d = rng.choice([8, 16, 32, 64, 80, 128, 30])
        right = ZM.delta(G * rng.choice([1, 2]), G, d, rng.choice([d, d, 16, 64, 96, 20]), rng.choice([1, 2, 3, 4, 5]))
        return left, right, rng.choice([1.0, 0.6, 1.3]), rng.choice([1.0, 0.5, 1.2])

    def ff():
        if rng.random() < 0.1:
            return None
        E = rng.choice([2, 4, 8, 12, 33])
        return ZM.moe(rng.choice([24, 64, 40, 17]), E, min(E, rng.choice([1, 2, 3, 4])), rng.choice([None, 32, 72, 128, 19]))

    layers, owners = [], []
    for i in range(rng.randint(3, 6)):
        if owners and rng.random() < 0.4:             # a reader of an earlier layer's keys
            j = rng.choice(owners)
            m = copy.deepcopy(layers[j]["mixer"])
            m.pop("mask", None)
            w = rng.choice(WINDOWS)
            if w:
                m["mask"] = {"size": w}
            m.update(kv_from=j, heads=m["kv_heads"] * rng.choice([1, 2, 4]), scale=rng.choice([0.1, 0.25]))
            layers.append(ZM.one(m, ff()))
        elif rng.random() < 0.5:
            owners.append(i)
            layers.append(ZM.one(attention(), ff()))
        else:
            left, right, a, b = pair()
            layers.append(ZM.two(left, right, ff(), a, b))
    return ZM.model(rng.choice([97, 300, 1000, 450]), rng.choice([64, 100, 128, 96, 328]), layers,
                    scale=rng.choice([1.0, 4.0, 11.3]), side=rng.choice([None, 8, 24, 13]),
                    eps=rng.choice([1e-5, 1e-6]))


@pytest.mark.parametrize("seed", range(12))
def test_a_random_configuration(tmp_path, seed):
    """Three unequal requests in one batch, prompts with every logit wanted, then decoded together
    while the shorter ones end, in both precisions."""
    rng = random.Random(seed)
    cfg = random_config(rng)
    P = ZM.make_tensors(cfg, seed, (rng.choice([4, 8, 16, 5]), rng.choice([4, 8, 16, 9])))
    folder = ZM.write_model(tmp_path / "m", cfg, P)
    lens = [rng.choice([300, 140, 70]), rng.choice([1, 9, 66]), rng.choice([130, 200])]
    heads = [max(1, n - rng.choice([3, 20, 40])) for n in lens]
    seqs = [_tokens(cfg["vocab"], n, 100 * seed + i) for i, n in enumerate(lens)]
    for dtype in DTYPES:
        e = _engine(folder, dtype)
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
            assert_close(torch.cat(got[i]), _plain(e, slots[i], seqs[i], P, cfg, dtype), dtype,
                         f"request {i}; {cfg}")
