"""Bumulix's mechanisms alone on the GPU, each against its plain restatement in float64, with
inputs made so that a fault shows: a query whose one map points at one key (far away, at a page's
end, just inside and just outside a window), keys told apart by their rotated part alone, pages an
earlier owner filled with NaN, streams of very different sizes."""
import math

import pytest
import torch

import plain_bumulix as PB
from nimbus_infer_rs_b200.cache import SequenceCache
from nimbus_infer_rs_b200.csrc import ops as ops_mod
from nimbus_infer_rs_b200.engine.batch import build_layout
from nimbus_infer_rs_b200.parts.base import KVRequest
from nimbus_infer_rs_b200.parts.rotary import rotary_frequencies

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
ACT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
TOL = {"float32": 2e-5, "bfloat16": 2e-2}
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module", autouse=True)
def _few_threads():
    """The plain implementation's matrices are small: many threads only wait for one another."""
    n = torch.get_num_threads()
    torch.set_num_threads(2)
    yield
    torch.set_num_threads(n)


@pytest.fixture(scope="module")
def ops():
    return ops_mod.backend()


def _rnd(*shape, seed=0, s=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * s


def _close(got, ref, tol, what=""):
    got, ref = got.double().cpu(), ref.double().cpu()
    assert got.shape == ref.shape, what
    assert torch.isfinite(got).all(), what
    err = float((got - ref).abs().max())
    assert err <= tol * max(float(ref.abs().max()), 1e-30), f"{what}: {err:.3e}"


# ----------------------------------------------------------------------------- streams
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S", [1, 2, 3, 4, 5, 8])
@pytest.mark.parametrize("n,d", [(3, 1), (9, 7), (5, 56), (70, 256), (700, 1024), (2, 4100), (601, 2050)])
def test_streams_written_back_and_read(ops, dtype, S, n, d):
    """Streams of very different sizes: one taken for another is far off."""
    sizes = torch.tensor([3.0 ** i for i in range(S)])
    xs = (_rnd(S, n, d, seed=1) * sizes[:, None, None]).double()
    y, ls, gamma = _rnd(n, d, seed=2).double(), _rnd(d, seed=3).double(), _rnd(d, seed=4).double() + 1.0
    mix, gain, coef = _rnd(S, S, seed=5).double(), _rnd(S, seed=6).double(), _rnd(S, seed=7).double()

    def dev(t):
        return t.float().contiguous().to(DEV)

    def rows(t):          # [S, n, d] -> [n, S * d]
        return t.transpose(0, 1).reshape(n, S * d)

    new = PB.write_streams(xs, mix, gain, ls * y, 1.0)
    write = (dev(y), dev(ls), dev(mix), dev(gain))
    read = (dev(coef), dev(gamma), 3e-4)
    # read alone
    out = torch.empty(n, d, device=DEV, dtype=ACT[dtype])
    x = dev(rows(xs))
    ops.streams(x, S, False, read=read, out=out)
    _close(out, PB.plain_norm(PB.read_streams(xs, coef), gamma, 3e-4), TOL[dtype] / 2, "read")
    # write-back in place, with and without a read
    ops.streams(x, S, False, write=write, into=x, read=read, out=out)
    _close(x, rows(new), 2e-6, "streams")
    _close(out, PB.plain_norm(PB.read_streams(new, coef), gamma, 3e-4), TOL[dtype] / 2, "read after write")
    x = dev(rows(xs))
    ops.streams(x, S, False, write=write, into=x)
    _close(x, rows(new), 2e-6, "streams without a read")
    # the sum alone: the streams are not stored
    x, total = dev(rows(xs)), torch.empty(n, d, device=DEV)
    before = x.clone()
    ops.streams(x, S, False, write=write, total=total)
    assert torch.equal(x, before)
    _close(total, new.sum(0), 1e-5, "sum")
    # from the single row that all streams equal
    one = dev(xs[0])
    same = torch.stack([xs[0].float().double()] * S)
    into = torch.full((n, S * d), 9.0, device=DEV)
    ops.streams(one, S, True, read=read, out=out)
    _close(out, PB.plain_norm(PB.read_streams(same, coef), gamma, 3e-4), TOL[dtype] / 2, "first read")
    ops.streams(one, S, True, write=write, into=into, read=read, out=out)
    _close(into, rows(PB.write_streams(same, mix, gain, ls * y, 1.0)), 2e-6, "first streams")


def test_bounded_logits(ops):
    x = _rnd(7, 333, seed=1, s=40.0)
    for cap in (0.5, 30.0):
        got = x.to(DEV)
        ops.softcap_rows(got, cap)
        _close(got, PB.capped(x.double(), cap), 1e-6, f"cap {cap}")
        assert float(got.abs().max()) <= cap


# ----------------------------------------------------------------------------- differential attention
def _stores(dtype, G, d2, dv, tokens, window=0, fill=None):
    shared = d2 == dv
    cache = SequenceCache({0: KVRequest(G, d2, window, 2 if shared else 1)}, {}, cache_tokens=tokens,
                          max_seq_len=tokens, dtype=ACT[dtype], device=torch.device(DEV), n_slots=4,
                          extra_kv_requests={} if shared else {(0, 0): KVRequest(G, dv, window, 1)})
    if fill is not None:           # what an earlier owner of the pages left behind
        for g in cache.groups:
            g.storage.fill_(fill)
    keys = cache.layer_kv(0)
    return cache, keys, keys if shared else cache.layer_kv((0, 0))


def _plain(q, k, v, window, scale, lam, diff, eps):
    T = q.shape[0]
    see = PB.sees_window(T, window) if window else PB.sees_past(T)
    a = PB.two_maps(q.double(), k.double(), v.double(), see, scale)
    return PB.difference_of_maps(a[:, :, 0], a[:, :, 1], lam, diff, eps).reshape(T, -1)


def _run_rows(ops, dtype, fused, lay, keys, values, H, G, d2, dv, window, scale, lam, diff, eps):
    n = lay.n_rows
    qo = torch.empty(n, H * d2, device=DEV, dtype=ACT[dtype])
    ops.qkv_norm_rope_append(fused, 0, H * d2, H * d2 + G * d2, None, None, 0.0, None, 0, 1.0, lay, keys,
                             values, H, dv, qo, True)
    out = torch.full((n, H * dv), 7.0, device=DEV, dtype=ACT[dtype])
    ops.attention_differential(qo, lay, keys, values, H, out, scale, window, lam, 1.0 - diff, eps)
    return out


def _attention(ops, dtype, q, k, v, pieces, window=0, scale=1.0, lam=0.5, diff=0.3, eps=1e-5, fill=None):
    """One sequence cut into ``pieces``; q [T, H, 2, d], k [T, G, 2, d], v [T, G, dv] (fp32)."""
    T, H, _, d = q.shape
    G, dv = k.shape[1], v.shape[2]
    cache, keys, values = _stores(dtype, G, 2 * d, dv, T + 64, window, fill)
    fused = torch.cat([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], 1)
    fused = torch.cat([fused, torch.zeros(T, -fused.shape[1] % 8)], 1).to(DEV)
    slot = cache.alloc_slot()
    outs, at = [], 0
    for n in pieces:
        cache.reserve([(slot, n)])
        lay = build_layout([(slot, [1] * n, [])], [at], torch.device(DEV))
        outs.append(_run_rows(ops, dtype, fused[at:at + n].contiguous(), lay, keys, values, H, G, 2 * d,
                              dv, window, scale, lam, diff, eps).float().cpu())
        cache.advance(slot, n)
        at += n
    ops.raise_device_errors()
    return torch.cat(outs)


SHAPES = [  # H, G, d, dv, window, lam, diff
    (4, 2, 12, 20, 9, 0.6, 0.4),
    (4, 2, 32, 64, 100, 0.7, 0.5),
    (4, 1, 32, 64, 0, 0.3, 0.5),
    (2, 1, 64, 128, 64, 0.9, 0.8),
    (8, 2, 64, 128, 130, 0.55, 0.6),
    (6, 2, 64, 128, 0, 0.8, 0.6),
    (3, 3, 16, 32, 70, 1.2, -0.2),
    (16, 2, 16, 32, 65, 0.4, 0.2),      # too many maps a key head for the decode kernel
    (2, 2, 64, 64, 96, 0.5, 0.1),       # values of another size than two keys
    (2, 1, 40, 128, 0, 0.5, 0.1),
    (5, 5, 24, 48, 200, 0.5, 0.1),
    (2, 1, 128, 256, 90, 0.5, 0.1),
    (1, 1, 1, 2, 1, 0.2, 0.3),
    (3, 1, 7, 14, 0, -0.4, 0.3),        # the second map is added
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", range(len(SHAPES)))
def test_attention_whole_in_portions_and_token_by_token(ops, dtype, shape):
    H, G, d, dv, window, lam, diff = SHAPES[shape]
    T = 275
    q, k, v = _rnd(T, H, 2, d, seed=1), _rnd(T, G, 2, d, seed=2), _rnd(T, G, dv, seed=3)
    kw = dict(window=window, scale=1.5 / math.sqrt(d), lam=lam, diff=diff, eps=1e-5)
    if window == 1:       # a token sees itself: the difference is (1 - lam) of its own value
        kw["eps"] = 1e-2
    ref = _plain(q, k, v, **kw)
    for pieces in ((T,), (2, 61, 1, 2, 64, 3, 142), (202,) + (1,) * 73):
        got = _attention(ops, dtype, q, k, v, pieces, fill=float("nan"), **kw)
        _close(got, ref, TOL[dtype], f"shape {shape} in pieces {pieces[:3]}")
    if dtype == "bfloat16" and dv == 2 * d and d in (32, 64):
        # the same heads on the mma.sync prompt kernel, which takes them when tcgen05 is off
        ops.use_tcgen05 = False
        try:
            got = _attention(ops, dtype, q, k, v, (2, 61, 1, 2, 64, 3, 142), fill=float("nan"), **kw)
        finally:
            ops.use_tcgen05 = True
        _close(got, ref, TOL[dtype], f"shape {shape} without tcgen05")


@pytest.mark.parametrize("d", [32, 64])
def test_scores_that_grow_along_the_keys(ops, d):
    """Every key's score is far above those before it, in one map rising and in the other falling:
    the exponents' reference moves at every turn, or never, and a result that is not rescaled with
    it is far off."""
    T, H, G = 700, 2, 1
    q, k, v = _rnd(T, H, 2, d, seed=1, s=0.1), _rnd(T, G, 2, d, seed=2, s=0.1), _rnd(T, G, 2 * d, seed=3)
    q[:, :, :, 0] = 1.0
    ramp = torch.linspace(0.0, 60.0, T).bfloat16().float()[:, None]
    k[:, :, 0, 0], k[:, :, 1, 0] = ramp, ramp.flip(0)
    for window in (0, 300):
        kw = dict(window=window, scale=1.0, lam=0.5, diff=0.3, eps=1e-5)
        ref = _plain(q, k, v, **kw)
        for pieces in ((T,), (130, 570)):
            _close(_attention(ops, "bfloat16", q, k, v, pieces, **kw), ref, TOL["bfloat16"], f"{window} {pieces}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d,dv", [(16, 32), (32, 64), (64, 128), (64, 64), (20, 16)])
def test_a_key_just_inside_and_just_outside_for_either_map(ops, dtype, d, dv):
    """The query at ``at`` and the key at ``to`` share one large direction in one of the two maps;
    the first number of the values marks ``to``.  Seen by the first map it makes that number
    positive, by the second negative, beyond the window's edge it leaves zero."""
    H, G, T = 2, 1, 330
    for window in (64, 65, 130, 0):
        for at in (T - 3, 129):
            for to in ((at - window + 1, at - window, at) if window else (0, 63, 64, at)):
                for a in (0, 1):
                    q, k = _rnd(T, H, 2, d, seed=at, s=0.03), _rnd(T, G, 2, d, seed=to + 1, s=0.03)
                    v = torch.zeros(T, G, dv)
                    v[:, :, 1] = 0.25
                    v[to, :, 0] = 1.0
                    q[at, :, a, -1] += 6.0
                    k[to, :, a, -1] += 6.0
                    seen = not window or at - to < window
                    for pieces in ((T,), (at - 2, 1, 1, 1, 1, T - at - 2), (to + 1, T - to - 1)):
                        if sum(pieces) != T or min(pieces) < 1:
                            continue
                        got = _attention(ops, dtype, q, k, v, pieces, window=window, lam=0.5)
                        x = float(got[at, 0])
                        where = (window, at, to, a, pieces[:3], x)
                        if not seen:
                            assert x == 0.0, where
                        else:
                            assert (x > 1.0) if a == 0 else (x < -1.0), where


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d,dv", [(32, 64), (24, 16)])
def test_an_unequal_batch_against_each_alone(ops, dtype, d, dv):
    H, G, window = 4, 2, 70
    lens, heads = (250, 9, 70), (240, 1, 66)
    cache, keys, values = _stores(dtype, G, 2 * d, dv, 8 * 64)
    data = [(_rnd(n, H, 2, d, seed=10 + i), _rnd(n, G, 2, d, seed=20 + i), _rnd(n, G, dv, seed=30 + i))
            for i, n in enumerate(lens)]
    fused = [torch.cat([t.reshape(n, -1) for t in ts], 1).to(DEV) for ts, n in zip(data, lens)]
    slots = [cache.alloc_slot() for _ in lens]
    got = [[] for _ in lens]

    def step(parts):      # parts: (sequence, start, count)
        cache.reserve([(slots[i], n) for i, _, n in parts])
        lay = build_layout([(slots[i], [1] * n, []) for i, _, n in parts], [a for _, a, _ in parts],
                           torch.device(DEV), pad_rows_to=8)
        rows = torch.zeros(lay.n_rows, fused[0].shape[1], device=DEV)
        r = 0
        for i, a, n in parts:
            rows[r:r + n] = fused[i][a:a + n]
            r += n
        out = _run_rows(ops, dtype, rows, lay, keys, values, H, G, 2 * d, dv, window, 0.2, 0.6, 0.5, 1e-5)
        r = 0
        for i, a, n in parts:
            got[i].append(out[r:r + n].float().cpu())
            cache.advance(slots[i], n)
            r += n
        assert r == lay.n_rows or float(out[r:].abs().max()) == 0.0       # padding rows

    step([(i, 0, h) for i, h in enumerate(heads)])
    k = 0
    while True:
        live = [(i, heads[i] + k, 1) for i in range(3) if heads[i] + k < lens[i]]
        if not live:
            break
        step(live)
        k += 1
    for i, (q, kk, v) in enumerate(data):
        _close(torch.cat(got[i]), _plain(q, kk, v, window, 0.2, 0.6, 0.5, 1e-5), TOL[dtype], f"sequence {i}")


# ----------------------------------------------------------------------------- latent attention
def _latent(ops, dtype, cq_rows, down, gamma, H, R, rot, dims, base, scaling, pieces, scale, eps=1e-5, fill=None):
    """Attention over the cached rows: ``cq_rows`` = (queries in the latent's space [T, H, R], their
    rotated parts [T, H, rot]), ``down`` [T, R + rot]; returns [T, H, R]."""
    a0, qr = cq_rows
    T = down.shape[0]
    cache = SequenceCache({0: KVRequest(1, R + rot, 0, 1)}, {}, cache_tokens=T + 64, max_seq_len=T + 64,
                          dtype=ACT[dtype], device=torch.device(DEV), n_slots=2)
    if fill is not None:
        for g in cache.groups:
            g.storage.fill_(fill)
    kv = cache.layer_kv(0)
    freq, amp = rotary_frequencies(dims, base, scaling)
    freq = freq.to(DEV)
    src = torch.cat([torch.zeros(T, 3), down, torch.zeros(T, 2)], 1).to(DEV)
    qs = torch.cat([torch.zeros(T, 5), qr.reshape(T, -1)], 1).to(DEV)
    slot = cache.alloc_slot()
    outs, at = [], 0
    for n in pieces:
        cache.reserve([(slot, n)])
        lay = build_layout([(slot, [1] * n, [])], [at], torch.device(DEV))
        a = torch.empty(n, H, R + rot, device=DEV, dtype=ACT[dtype])
        a[:, :, :R] = a0[at:at + n].to(DEV).to(ACT[dtype])
        a = a.view(n, -1)
        ops.latent_rope_append(src[at:at + n].contiguous(), 3, gamma.to(DEV), eps, freq, rot, dims, amp,
                               qs[at:at + n].contiguous(), 5, a, H, lay, kv, True)
        out = torch.empty(n, H * R, device=DEV, dtype=ACT[dtype])
        ops.attention_latent(a, lay, kv, H, None, out, scale, 0, R)
        cache.advance(slot, n)
        outs.append(out.float().cpu())
        at += n
    return torch.cat(outs).view(T, H, R)


def _latent_plain(a0, qr, down, gamma, R, dims, base, scaling, scale, eps=1e-5):
    a0, qr, down = a0.double(), qr.double(), down.double()
    c = PB.plain_norm(down[:, :R], gamma.double(), eps)
    kr = PB.turned(down[:, R:], dims, base, scaling)
    qr = PB.turned(qr, dims, base, scaling)
    T, H = a0.shape[:2]
    out = torch.zeros(T, H, R, dtype=torch.float64)
    for h in range(H):
        s = (a0[:, h] @ c.T + qr[:, h] @ kr.T) * scale
        out[:, h] = PB.weights_over(s, PB.sees_past(T)) @ c
    return out


YARN = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 0.5}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,R,rot,dims,scaling", [
    (3, 20, 6, 6, YARN), (4, 64, 16, 16, None), (16, 256, 64, 64, YARN), (5, 96, 40, 24, YARN),
    (1, 72, 8, 8, YARN), (2, 128, 64, 64, None), (3, 16, 72, 72, YARN), (20, 40, 32, 32, YARN),
    (1, 1, 2, 2, None), (2, 192, 48, 48, YARN)])
def test_latent_rows_with_a_rotated_part(ops, dtype, H, R, rot, dims, scaling):
    T = 203
    a0, qr = _rnd(T, H, R, seed=1), _rnd(T, H, rot, seed=2)
    down, gamma = _rnd(T, R + rot, seed=3), _rnd(R, seed=4, s=0.2) + 1.0
    scale = 1.0 / math.sqrt(R + rot)
    ref = _latent_plain(a0, qr, down, gamma, R, dims, 200.0, scaling, scale)
    for pieces in ((T,), (2, 61, 1, 2, 64, 3, 70), (130,) + (1,) * 73):
        got = _latent(ops, dtype, (a0, qr), down, gamma, H, R, rot, dims, 200.0, scaling, pieces, scale,
                      fill=float("nan"))
        _close(got, ref, TOL[dtype], f"pieces {pieces[:3]}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("R,rot", [(32, 16), (96, 32), (128, 64), (12, 6)])
def test_a_key_found_by_its_rotated_part_alone(ops, dtype, R, rot):
    """All latents equal but for one marked number; the query's latent part is zero and its rotated
    part, turned, meets the rotated part of one key only: a rotation that is off by a position, or
    an amplitude left out, loses it.  The slow pairs carry the direction, so distance matters
    little."""
    T, H = 330, 2
    for at, to in ((T - 1, 0), (T - 1, 63), (T - 1, 64), (300, 299), (129, 127), (200, 200)):
        down = torch.zeros(T, R + rot)
        down[:, 0] = 1.0
        down[:, 1] = -1.0
        down[to, 1] = 1.0
        down[to, R + rot // 2 - 1] = 5.0       # the slowest pair: (rot/2 - 1, rot - 1)
        a0, qr = torch.zeros(T, H, R), torch.zeros(T, H, rot)
        qr[at, :, rot // 2 - 1] = 5.0
        gamma = torch.ones(R)
        ref = _latent_plain(a0, qr, down, gamma, R, rot, 1e6, YARN, 1.0)
        assert float(ref[at, 0, 1]) > 0.97 * float(ref[at, 0, 0])       # it stands out
        for pieces in ((T,), (at - 1, 1, 1, T - at - 1) if at + 1 < T else (at, 1), (to + 1, T - to - 1)):
            if sum(pieces) != T or min(pieces) < 1:
                continue
            got = _latent(ops, dtype, (a0, qr), down, gamma, H, R, rot, rot, 1e6, YARN, pieces, 1.0)
            _close(got[at], ref[at], TOL[dtype], f"{at} -> {to} in {pieces[:3]}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,H,n_in,n_out,gap", [(3, 4, 16, 24, 8), (100, 3, 32, 64, 0), (70, 5, 7, 9, 3), (17, 2, 128, 80, 16)])
def test_map_per_head_with_a_gate_on_every_number(ops, dtype, n, H, n_in, n_out, gap):
    x, w = _rnd(n, H * n_in + 8, seed=1), _rnd(H, n_out, n_in, seed=2)
    gate = _rnd(n, 5 + H * n_out, seed=3, s=2.0)
    lay = build_layout([(0, [1] * n, [])], [0], torch.device(DEV))
    out = torch.full((n, H * (n_out + gap)), 9.0, device=DEV, dtype=ACT[dtype])
    wd = w.to(ACT[dtype]).to(DEV)
    ops.head_linear(x.to(DEV), 8, wd, out, lay, gate=gate.to(DEV), gate_col=5, gate_each=True,
                    out_stride=n_out + gap)
    xs = x[:, 8:].view(n, H, n_in).double()
    ref = torch.einsum("rhi,hoi->rho", xs, w.to(ACT[dtype]).double())
    ref = ref * torch.sigmoid(gate[:, 5:].view(n, H, n_out).double())
    got = out.float().cpu().view(n, H, n_out + gap)
    _close(got[:, :, :n_out], ref, TOL[dtype], "gated")
    assert gap == 0 or bool((got[:, :, n_out:] == 9.0).all())           # what lies between is left alone
