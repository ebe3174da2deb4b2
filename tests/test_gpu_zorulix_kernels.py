"""Zorulix's mechanisms alone on the GPU, each against its plain restatement in float64, with
inputs made so that a fault shows: a query that points at one key (far away, at a page's end, just
inside and just outside a window), norms over heads of very different sizes, decays that are
almost one and decays that leave nothing, pages an earlier owner filled with NaN."""
import math

import pytest
import torch

import plain_zorulix as PZ
from nimbus_infer_rs_b200.cache import SequenceCache
from nimbus_infer_rs_b200.csrc import ops as ops_mod
from nimbus_infer_rs_b200.csrc.ops import ACT_SILU
from nimbus_infer_rs_b200.engine.batch import build_layout
from nimbus_infer_rs_b200.parts.base import KVRequest, StateRequest
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


def _layout(parts, starts, pad=1):
    return build_layout([(s, [1] * n, []) for s, n in parts], starts, torch.device(DEV), pad_rows_to=pad) \
        if pad > 1 else build_layout([(s, [1] * n, []) for s, n in parts], starts, torch.device(DEV))


# ----------------------------------------------------------------------------- row passes
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,d", [(1, 1), (5, 7), (9, 56), (70, 256), (3, 2048), (300, 3000), (2, 4100), (2, 8200)])
def test_two_results_scaled_into_the_stream(ops, dtype, n, d):
    a, b, x = _rnd(n, d, seed=1), _rnd(n, d, seed=2, s=5.0), _rnd(n, d, seed=3)
    gamma = _rnd(d, seed=4) + 1.0
    new = x.double() + 1.3 * a.double() - 0.4 * b.double()
    xd = x.to(DEV)
    out = torch.empty(n, d, device=DEV, dtype=ACT[dtype])
    ops.scaled_pair_add(a.to(DEV), 1.3, b.to(DEV), -0.4, xd, gamma.to(DEV), 3e-4, out)
    _close(xd, new, 2e-6, "stream")
    _close(out, PZ.over_rms(new, 3e-4) * gamma.double(), TOL[dtype] / 2, "next rows")
    xd = x.to(DEV)
    ops.scaled_pair_add(a.to(DEV), 1.3, b.to(DEV), -0.4, xd)
    _close(xd, new, 2e-6, "stream without a norm")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_gated_half_times_a_gate_per_row(ops, dtype):
    for n, d, gate in ((3, 5, 21), (70, 40, 0), (9, 128, 300)):
        x = _rnd(n, 310, seed=n)
        x[:, gate] = torch.linspace(-6, 6, n)
        out = torch.empty(n, d, device=DEV, dtype=ACT[dtype])
        ops.glu_rows(x.to(DEV), 1, 150, ACT_SILU, out, 0.0, gate)
        xx = x.double()
        _close(out, PZ.silu(xx[:, 1:1 + d]) * xx[:, 150:150 + d] * torch.sigmoid(xx[:, gate:gate + 1]),
               TOL[dtype] / 2)


@pytest.mark.parametrize("E,top", [(1, 1), (5, 5), (12, 3), (33, 4), (64, 8), (200, 3), (300, 2)])
def test_router_with_a_bias_and_weights_over_the_chosen(ops, E, top):
    n = 37
    lay = _layout([(0, n)], [0])
    z, bias = _rnd(n, E + 6, seed=E, s=3.0), _rnd(E, seed=E + 1, s=4.0)
    z[0, 4:4 + E] += 90.0                          # far from zero: the softmax must not overflow
    idx = torch.empty(n, top, device=DEV, dtype=torch.int32)
    w = torch.empty(n, top, device=DEV)
    ops.moe_route(z.to(DEV), 4, E, top, True, lay, idx, w, bias.to(DEV))
    want_idx, want = PZ.chosen(z[:, 4:4 + E].double() + bias.double(), top)
    assert torch.equal(idx.cpu().long(), want_idx)
    _close(w, want, 2e-6)
    assert torch.allclose(w.sum(1).cpu(), torch.ones(n), atol=1e-5)


def test_experts_results_added_and_the_stream_rounded(ops):
    n, top, d = 9, 3, 50
    place = torch.randperm(n * top, generator=torch.Generator().manual_seed(1)).to(torch.int32)
    y, w, x = _rnd(n * top, d, seed=2), _rnd(n, top, seed=3), _rnd(n, d, seed=4)
    new = x.double() + (w.double()[:, :, None] * y.double()[place.long()].view(n, top, d)).sum(1)
    for dtype in DTYPES:
        xd, out = x.to(DEV), torch.empty(n, d, device=DEV, dtype=ACT[dtype])
        ops.moe_combine(y.to(DEV), place.to(DEV), w.to(DEV), xd, out)
        _close(xd, new, 2e-6)
        assert torch.equal(out, xd.to(ACT[dtype]))


@pytest.mark.parametrize("n", [1, 5, 16, 17, 200])
@pytest.mark.parametrize("rank,width", [(8, 24), (16, 130), (64, 512)])
def test_two_low_rank_maps_as_one_product(ops, n, rank, width):
    lay = _layout([(0, n)], [0])
    x, w = _rnd(n, 40 + 2 * rank, seed=n), _rnd(2, width, rank, seed=2, s=rank ** -0.5).to(torch.bfloat16)
    out = torch.empty(n, 2 * width, device=DEV)
    ops.head_linear(x.to(DEV), 32, w.to(DEV), out, lay)
    xs = x[:, 32:32 + 2 * rank].to(torch.bfloat16).double().view(n, 2, rank)
    _close(out, torch.einsum("nhr,hor->nho", xs, w.double()).reshape(n, -1), 2e-5)
    ops.head_linear(x.to(DEV), 32, w.float().to(DEV), out, lay)             # the 32-bit run's
    xs = x[:, 32:32 + 2 * rank].double().view(n, 2, rank)
    _close(out, torch.einsum("nhr,hor->nho", xs, w.double()).reshape(n, -1), 2e-6)


# ----------------------------------------------------------------------------- attention
def _store(dtype, G, d, dv, tokens, window=0, fill=None):
    cache = SequenceCache({0: KVRequest(G, d, window, value_dim=None if d == dv else dv)}, {},
                          cache_tokens=tokens, max_seq_len=tokens, dtype=ACT[dtype],
                          device=torch.device(DEV), n_slots=4)
    if fill is not None:           # what an earlier owner of the pages left behind
        for g in cache.groups:
            g.storage.fill_(fill)
    return cache


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,dv,rot", [(4, 2, 12, 20, 12), (6, 3, 64, 64, 32), (3, 1, 300, 8, 300),
                                          (8, 2, 48, 96, 48), (1, 1, 2, 1, 2), (5, 5, 7, 7, 0)])
def test_norms_over_all_heads_then_rotation(ops, dtype, H, G, d, dv, rot):
    """Heads of very different sizes: a norm per head would be far off."""
    T, eps, pos0 = 9, 1e-5, 60                           # across a page's end
    sizes = torch.tensor([3.0 ** (i % 4) for i in range(H)])
    q, k, v = _rnd(T, H, d, seed=1) * sizes[:, None], _rnd(T, G, d, seed=2) * sizes[:G, None], _rnd(T, G, dv, seed=3)
    wq, wk = _rnd(H * d, seed=4) + 1.0, _rnd(G * d, seed=5) + 1.0
    scaling = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 0.5}
    turn = {"dims": rot, "base": 300.0, "scaling": scaling} if rot else None
    freq, amp = rotary_frequencies(rot, 300.0, scaling) if rot else (None, 1.0)
    cache = _store(dtype, G, d, dv, 128)
    slot = cache.alloc_slot()
    cache.reserve([(slot, pos0 + T)])
    lay = _layout([(slot, T)], [pos0])
    fused = torch.cat([torch.zeros(T, 3), q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], 1).to(DEV)
    kv = cache.layer_kv(0)
    q_out = torch.empty(T, H * d, device=DEV, dtype=ACT[dtype])
    cols = (3, 3 + H * d, 3 + (H + G) * d)
    fq = freq.to(DEV) if rot else None
    ops.qkv_norm_rope_append(fused, *cols, wq.to(DEV), wk.to(DEV), eps, fq, rot, amp, lay, kv, kv, H, dv,
                             q_out, True, True)

    def plain(x, w, heads):
        x = (PZ.over_rms(x.double().reshape(T, -1), eps) * w.double()).view(T, heads, d)
        return PZ.rotated(torch.cat([x.new_zeros(pos0, heads, d), x]), turn)[pos0:]
    _close(q_out.view(T, H, d), plain(q, wq, H), TOL[dtype], "queries")
    pages = kv.block_table[slot].long()

    def cached(plane):
        return torch.stack([plane[pages[p // 64], :, p % 64] for p in range(pos0, pos0 + T)])
    _close(cached(kv.k), plain(k, wk, G), TOL[dtype], "keys")
    _close(cached(kv.v), v, TOL[dtype], "values")
    # queries alone: the store stays as it is
    before = kv.k.clone(), kv.v.clone()
    q_two = torch.empty_like(q_out)
    ops.qkv_norm_rope_append(fused[:, :3 + H * d].contiguous(), 3, 0, 0, wq.to(DEV), None, eps, fq, rot, amp,
                             lay, kv, kv, H, dv, q_two, False, True)
    assert torch.equal(q_two, q_out)
    assert torch.equal(kv.k, before[0]) and torch.equal(kv.v, before[1])


def _attend(ops, dtype, q, k, v, pieces, window, scale, sink, fill=None, cache=None, trim=True):
    """One sequence cut into ``pieces``; q [T, H, d], k [T, G, d], v [T, G, dv] (fp32)."""
    T, H, d = q.shape
    G, dv = k.shape[1], v.shape[2]
    cache = cache or _store(dtype, G, d, dv, T + 64, window if trim else 0, fill)
    kv = cache.layer_kv(0)
    fused = torch.cat([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], 1).to(DEV)
    zero = torch.zeros(H, device=DEV) if sink else None
    slot, outs, at = cache.alloc_slot(), [], 0
    for n in pieces:
        cache.reserve([(slot, n)])
        lay = _layout([(slot, n)], [at])
        qo = torch.empty(n, H * d, device=DEV, dtype=ACT[dtype])
        ops.qkv_norm_rope_append(fused[at:at + n].contiguous(), 0, H * d, (H + G) * d, None, None, 0.0, None, 0,
                                 1.0, lay, kv, kv, H, dv, qo, True)
        out = torch.full((n, H * dv), 7.0, device=DEV, dtype=ACT[dtype])
        ops.attention_masked(qo, lay, kv, kv, H, zero, out, scale, 0.0, window)
        outs.append(out.float().cpu())
        cache.advance(slot, n)
        at += n
    ops.raise_device_errors()
    cache.free_slot(slot)
    return torch.cat(outs)


SHAPES = [  # H, G, d, dv, window, sink
    (4, 2, 12, 20, 9, True),
    (8, 1, 48, 96, 136 - 6, False),
    (4, 2, 64, 128, 64, True),
    (4, 2, 32, 64, 65, False),
    (3, 3, 128, 64, 100, True),
    (2, 1, 96, 128, 0, False),
    (2, 2, 24, 16, 1, True),
    (6, 1, 40, 56, 63, False),
    (16, 1, 16, 48, 128, True),        # more query heads over a key head than the decode kernel takes
    (2, 1, 72, 8, 200, False),
    (2, 1, 130, 30, 70, True),         # beyond the tensor-core kernels
    (4, 2, 64, 64, 96, True),
    (4, 1, 128, 128, 65, True),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", SHAPES, ids=lambda s: "x".join(map(str, s)))
def test_attention_over_keys_and_values_of_their_own_sizes(ops, dtype, shape):
    """Whole prompts, portions and single tokens on pages that held NaN."""
    H, G, d, dv, window, sink = shape
    T = 210
    q, k, v = (x.to(torch.bfloat16).float() for x in (_rnd(T, H, d, seed=1), _rnd(T, G, d, seed=2), _rnd(T, G, dv, seed=3)))
    scale = 1.5 * d ** -0.5
    ref = PZ.attend(q.double(), k.double(), v.double(), PZ.sees(T, window), scale, sink).reshape(T, -1)
    for pieces in ([T], [1] * 3 + [61, 1, 63, 2, 64] + [1] * 16, [130, 80]):
        assert sum(pieces) == T
        got = _attend(ops, dtype, q, k, v, pieces, window, scale, sink, fill=float("nan"))
        _close(got, ref, TOL[dtype] / (1 if dtype == "bfloat16" else 2), f"{pieces[:4]}...")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,dv,window", [(2, 1, 64, 128, 64), (2, 2, 32, 64, 65), (1, 1, 48, 96, 100),
                                             (2, 1, 128, 64, 130), (2, 1, 64, 64, 70), (1, 1, 20, 12, 33)])
def test_a_query_that_points_at_one_key(ops, dtype, H, G, d, dv, window):
    """The last row's score stands out at one key: just inside a window it decides the result,
    just outside it must not be seen; the same row computed in a prompt and as a single token."""
    T = 200
    for back in (0, 1, window - 1, window, window + 1, 63, 64, 65, T - 1 - 128, T - 1 - 127):
        if not 0 <= back < T:
            continue
        at = T - 1 - back
        q, k, v = _rnd(T, H, d, seed=1, s=0.1), _rnd(T, G, d, seed=2, s=0.1), _rnd(T, G, dv, seed=3)
        k[at] = 4.0 * torch.eye(d)[0]
        q[T - 1] = 4.0 * torch.eye(d)[0]
        v[at] = 5.0
        q, k, v = (x.to(torch.bfloat16).float() for x in (q, k, v))
        ref = PZ.attend(q.double(), k.double(), v.double(), PZ.sees(T, window), 1.0, True).reshape(T, -1)
        assert (float(ref[-1].min()) > 4.9) == (back < window)
        for pieces in ([T], [T - 1, 1], [T - 2, 2]):
            got = _attend(ops, dtype, q, k, v, pieces, window, 1.0, True)
            _close(got[-1:], ref[-1:], TOL[dtype], f"key {back} back, {pieces}")
            _close(got, ref, TOL[dtype], f"key {back} back, all rows")


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_sink_of_score_zero(ops, dtype):
    """Scores far below zero leave almost nothing of the values, scores far above hide the sink."""
    T, H, G, d, dv = 70, 2, 1, 16, 32
    base = torch.zeros(d)
    base[0] = 3.0
    for sign in (-1.0, 0.0, 1.0):
        q = base.expand(T, H, d).contiguous()
        k = (sign * base).expand(T, G, d).contiguous()
        v = _rnd(T, G, dv, seed=3).to(torch.bfloat16).float()
        for sink in (True, False):
            ref = PZ.attend(q.double(), k.double(), v.double(), PZ.sees(T, 9), 1.0, sink).reshape(T, -1)
            got = _attend(ops, dtype, q, k, v, [60, 1, 1, 8], 9, 1.0, sink)
            # with the sink and scores of -9 the results are tiny: compared on their own scale
            _close(got, ref, 2 * TOL[dtype], f"scores {9 * sign}, sink {sink}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d,dv", [(64, 128), (48, 96), (12, 20), (64, 64)])
def test_a_store_kept_for_the_longer_window_serves_both(ops, dtype, d, dv):
    """A writer with a window of 10 and readers of 5, 70 and without one over the same pages."""
    T, H, G = 190, 2, 1
    q, k, v = (x.to(torch.bfloat16).float() for x in (_rnd(T, H, d, seed=1), _rnd(T, G, d, seed=2), _rnd(T, G, dv, seed=3)))
    want = KVRequest(G, d, 10, value_dim=None if d == dv else dv)
    other = KVRequest(G, d, 70, value_dim=want.value_dim)
    assert want.covering(other).window == 70 and other.covering(want).window == 70
    assert want.covering(KVRequest(G, d, 0, value_dim=want.value_dim)).window == 0
    cache = SequenceCache({0: want.covering(other)}, {}, cache_tokens=4 * 64, max_seq_len=256,
                          dtype=ACT[dtype], device=torch.device(DEV), n_slots=2)
    kv = cache.layer_kv(0)
    fused = torch.cat([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], 1).to(DEV)
    slot, at, outs = cache.alloc_slot(), 0, {5: [], 10: [], 70: []}
    for n in (64, 30, 1, 1, 60, 1, 30, 1, 1, 1):
        cache.reserve([(slot, n)])
        lay = _layout([(slot, n)], [at])
        qo = torch.empty(n, H * d, device=DEV, dtype=ACT[dtype])
        ops.qkv_norm_rope_append(fused[at:at + n].contiguous(), 0, H * d, (H + G) * d, None, None, 0.0, None, 0,
                                 1.0, lay, kv, kv, H, dv, qo, True)
        for w, got in outs.items():
            out = torch.empty(n, H * dv, device=DEV, dtype=ACT[dtype])
            ops.attention_masked(qo, lay, kv, kv, H, None, out, 0.3, 0.0, w)
            got.append(out.float().cpu())
        cache.advance(slot, n)
        at += n
    for w, got in outs.items():
        ref = PZ.attend(q.double(), k.double(), v.double(), PZ.sees(T, w), 0.3, False).reshape(T, -1)
        _close(torch.cat(got), ref, TOL[dtype], f"window {w}")


# ----------------------------------------------------------------------------- the recurrence
def _recurrence_inputs(T, H, G, d, dv, seed, decay=0.0):
    """Rows [q | k | v], rate logits, decay and gate logits; ``decay``: added to the decay logits."""
    qkv = _rnd(T, 2 * G * d + H * dv, seed=seed)
    beta = _rnd(T, H + 5, seed=seed + 1, s=2.0)
    low = _rnd(T, 3 + H * (d + dv), seed=seed + 2, s=2.0)
    low[:, 3:3 + H * d] += decay
    return qkv, beta, low


def _weights(H, d, dv):
    return _rnd(H, seed=90, s=0.5), _rnd(H * d, seed=91, s=0.5) - 1.0, _rnd(dv, seed=92, s=0.2) + 1.0


def _plain_recurrence(qkv, beta, low, a_log, dt_bias, norm, H, G, d, dv, eps, S=None):
    T = qkv.shape[0]
    x = qkv.double()
    of = [h // (H // G) for h in range(H)]
    q = PZ.unit_vectors(x[:, :G * d].view(T, G, d)) * d ** -0.5
    k = PZ.unit_vectors(x[:, G * d:2 * G * d].view(T, G, d))
    g = torch.exp(-torch.exp(a_log.double())[:, None] *
                  PZ.softplus(low[:, 3:3 + H * d].double() + dt_bias.double()).view(T, H, d))
    o, S = PZ.delta_walk(q[:, of], k[:, of], x[:, 2 * G * d:].reshape(T, H, dv), g,
                         torch.sigmoid(beta[:, 2:2 + H].double()), S)
    o = PZ.over_rms(o, eps) * norm.double()
    return o.reshape(T, -1) * torch.sigmoid(low[:, 3 + H * d:].double()), S


def _run(ops, dtype, rows, weights, lay, state, H, G, d, dv, eps):
    qkv, beta, low = (r.to(DEV).contiguous() for r in rows)
    out = torch.full((lay.n_rows, H * dv), 7.0, device=DEV, dtype=ACT[dtype])
    ops.gated_delta(qkv, 0, None, 0, None, beta, 2, low, 3, 3 + H * d, *(w.to(DEV) for w in weights), eps, 1e-6, lay, state,
                    H, G, d, dv, out)
    return out.float().cpu()


RECURRENCES = [(1, 1, 1, 1), (2, 1, 3, 5), (4, 2, 9, 13), (3, 3, 32, 32), (2, 2, 33, 20), (4, 4, 64, 64),
               (2, 1, 64, 96), (2, 2, 128, 128), (1, 1, 100, 40), (3, 1, 128, 130), (2, 2, 129, 64),
               (1, 1, 256, 256), (2, 1, 200, 36), (20, 20, 64, 32)]


@pytest.mark.parametrize("H,G,d,dv", RECURRENCES)
def test_the_recurrence_whole_in_portions_and_token_by_token(ops, H, G, d, dv):
    """However the sequence is cut (blocks of eight tokens start anywhere), outputs and state."""
    T, eps = 75, 1e-5
    rows, weights = _recurrence_inputs(T, H, G, d, dv, 7), _weights(H, d, dv)
    ref, S = _plain_recurrence(*rows, *weights, H, G, d, dv, eps)
    n = H * d * dv
    pitch = -(-n // 4) * 4 + 4                     # state rows of another thing's numbers behind ours
    for pieces in ([T], [1] * T, [3, 1, 2, 5, 4, 1, 1, 30, 28], [2] * 37 + [1]):
        buf = torch.zeros(3, pitch, device=DEV)
        buf[:, n:] = 5.0
        state, got, at = buf[:, :n], [], 0
        for m in pieces:
            lay = _layout([(1, m)], [at])
            got.append(_run(ops, "float32", [r[at:at + m] for r in rows], weights, lay, state, H, G, d, dv, eps))
            at += m
        _close(torch.cat(got), ref, 5e-5, f"outputs, {pieces[:5]}")
        _close(state[1].view(H, d, dv), S, 2e-5, f"state, {pieces[:5]}")
        assert float(buf[0, :n].abs().max()) == 0.0 and float(buf[2, :n].abs().max()) == 0.0
        assert torch.equal(buf[:, n:], torch.full_like(buf[:, n:], 5.0))


@pytest.mark.parametrize("decay", [-12.0, 0.0, 4.0, 30.0, 300.0])
@pytest.mark.parametrize("d,dv", [(16, 24), (64, 64), (128, 128)])
def test_decays_of_every_strength(ops, decay, d, dv):
    """From almost nothing lost over the sequence to nothing left of the token before (decays that
    are zero in 32-bit): no step divides by a decay."""
    T, H, G, eps = 90, 2, 1, 1e-5
    rows, weights = _recurrence_inputs(T, H, G, d, dv, 3, decay), _weights(H, d, dv)
    ref, S = _plain_recurrence(*rows, *weights, H, G, d, dv, eps)
    for pieces in ([T], [40] + [1] * 50):
        state, got, at = torch.zeros(1, H * d * dv, device=DEV), [], 0
        for m in pieces:
            got.append(_run(ops, "float32", [r[at:at + m] for r in rows], weights, _layout([(0, m)], [at]),
                            state, H, G, d, dv, eps))
            at += m
        # few numbers are left of a strong decay's outputs before their norm: looser
        _close(torch.cat(got), ref, 3e-4, f"{pieces[:2]}")
        _close(state[0].view(H, d, dv), S, 2e-5, "state")


def test_a_token_far_back_is_remembered_or_forgotten(ops):
    """One key written at the start and read at the end, through one unit direction: with a decay
    of one it is still there, with a rate of one a second write replaces it."""
    H, G, d, dv, T = 1, 1, 64, 64, 201
    for again in (False, True):
        qkv = _rnd(T, 2 * d + dv, seed=1)
        qkv[:, d] = 0.0                                  # the keys between do not touch direction 0
        qkv[:, 2 * d:] *= 0.01
        first = torch.eye(d)[0]
        qkv[0, d:2 * d], qkv[0, 2 * d:] = 5.0 * first, 2.0
        if again:
            qkv[100, d:2 * d], qkv[100, 2 * d:] = 3.0 * first, -1.0
        qkv[T - 1, :d] = first
        beta = torch.full((T, 7), 40.0)
        low = torch.full((T, 3 + 2 * d), -60.0)          # decays of one
        low[:, 3 + d:] = 40.0
        weights = torch.zeros(H), torch.zeros(d), torch.ones(dv)
        ref, S = _plain_recurrence(qkv, beta, low, *weights, H, G, d, dv, 1e-5)
        assert float(S[0, 0].mean()) == pytest.approx(-1.0 if again else 2.0, rel=1e-3)
        for pieces in ([T], [T - 1, 1], [50, 51, 100]):
            state, got, at = torch.zeros(1, d * dv, device=DEV), [], 0
            for m in pieces:
                got.append(_run(ops, "float32", [r[at:at + m] for r in (qkv, beta, low)], weights,
                                _layout([(0, m)], [at]), state, H, G, d, dv, 1e-5))
                at += m
            _close(torch.cat(got)[-1:], ref[-1:], 1e-4, f"{pieces}")
            _close(state[0].view(H, d, dv), S, 2e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 64, 64), (2, 2, 128, 128), (3, 1, 20, 36)])
def test_unequal_sequences_in_one_batch(ops, dtype, H, G, d, dv):
    """Each against itself alone, on slots in any order; padding rows give zeros; then steps of one
    token with a sequence that has ended."""
    lens, slots, eps = [1, 37, 6, 64, 3], [4, 0, 3, 1, 2], 1e-5
    weights = _weights(H, d, dv)
    data = [_recurrence_inputs(n + 2, H, G, d, dv, 11 * i + 1) for i, n in enumerate(lens)]
    refs = [_plain_recurrence(*x, *weights, H, G, d, dv, eps)[0] for x in data]
    state = torch.zeros(6, H * d * dv, device=DEV)
    state[5] = 3.0
    lay = build_layout([(s, [1] * n, []) for s, n in zip(slots, lens)], [0] * 5, torch.device(DEV))
    rows = [torch.cat([x[j][:n] for x, n in zip(data, lens)]) for j in range(3)]
    got = _run(ops, dtype, rows, weights, lay, state, H, G, d, dv, eps)
    for g, ref, n in zip(torch.split(got, lens), refs, lens):
        _close(g, ref[:n], TOL[dtype], f"{n} tokens")
    assert torch.equal(state[5], torch.full_like(state[5], 3.0))
    for step in range(2):
        lay = build_layout([(s, [1], []) for s in slots], lens, torch.device(DEV))
        if step == 1:                                # sequence 2 has ended: a padding row
            lay.seq_slot[2] = -1
            lay.row_slot[2] = -1
        rows = [torch.stack([x[j][n + step] for x, n in zip(data, lens)]) for j in range(3)]
        before = state[slots[2]].clone()
        got = _run(ops, dtype, rows, weights, lay, state, H, G, d, dv, eps)
        for i, n in enumerate(lens):
            if step == 1 and i == 2:
                assert float(got[i].abs().max()) == 0.0 and torch.equal(state[slots[2]], before)
            else:
                _close(got[i], refs[i][n + step], TOL[dtype], f"{n} tokens and {step + 1}")


@pytest.mark.parametrize("H,G,d,dv", [(16, 16, 128, 128), (16, 8, 64, 96), (12, 4, 30, 130), (16, 2, 20, 33)])
def test_one_token_steps_of_many_heads(ops, H, G, d, dv):
    """Enough heads that a CTA takes all or 128 of a head's columns: twenty-four sequences, three
    tokens one by one, against each alone."""
    n, T, eps = 24, 3, 1e-5
    weights = _weights(H, d, dv)
    data = [_recurrence_inputs(T, H, G, d, dv, 5 * i) for i in range(n)]
    refs = [_plain_recurrence(*x, *weights, H, G, d, dv, eps) for x in data]
    state = torch.zeros(n, H * d * dv, device=DEV)
    slots = [(7 * i) % n for i in range(n)]
    for t in range(T):
        lay = build_layout([(s, [1], []) for s in slots], [t] * n, torch.device(DEV))
        rows = [torch.stack([x[j][t] for x in data]) for j in range(3)]
        got = _run(ops, "float32", rows, weights, lay, state, H, G, d, dv, eps)
        _close(got, torch.stack([ref[t] for ref, _ in refs]), 5e-5, f"token {t}")
    _close(state[slots].view(n, H, d, dv), torch.stack([S for _, S in refs]), 2e-5, "state")


@pytest.mark.parametrize("H,G,d,dv", [(2, 1, 12, 10), (2, 2, 12, 10), (3, 3, 64, 64), (2, 2, 128, 128),
                                      (2, 1, 64, 96), (1, 1, 129, 33), (4, 4, 20, 36)])
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
def test_convolution_and_recurrence_share_a_state_row(ops, taps, H, G, d, dv):
    """The matrices first, then the convolution's last inputs: a sequence cut anywhere goes on as
    if it had not been cut, alone and beside another, and the row of a slot that is used again
    starts from zeros."""
    T, eps = 40, 1e-5
    C, n = 2 * G * d + H * dv, H * d * dv
    raw, (_, beta, low), weights = _rnd(T, C, seed=1), _recurrence_inputs(T, H, G, d, dv, 2), _weights(H, d, dv)
    w = _rnd(C, taps, seed=3)
    ready = PZ.silu(PZ.causal_conv(raw.double(), w.double()))
    ref, _ = _plain_recurrence(ready, beta, low, *weights, H, G, d, dv, eps)
    want = -(-(n + (taps - 1) * C) // 4) * 4
    cache = SequenceCache({}, {0: StateRequest(want)}, cache_tokens=192, max_seq_len=64,
                          dtype=torch.float32, device=torch.device(DEV), n_slots=3)
    src = torch.cat([torch.full((T, 4), 9.0), raw, beta, torch.zeros(T, -(C + beta.shape[1]) % 4)], 1)
    for pieces in ([T], [1] * T, [2, 1, 3, 1, 1, 20, 12]):
        slot, beside, got, at = cache.alloc_slot(), cache.alloc_slot(), [], 0
        row = cache.layer_state(0)
        for m in pieces:
            # the neighbour: the sequence's first tokens again, one behind in every step
            lay = _layout([(beside, max(1, m - 1)), (slot, m)], [0, at])
            both = lambda x: torch.cat([x[:max(1, m - 1)], x[at:at + m]]).to(DEV).contiguous()
            out = torch.empty(lay.n_rows, H * dv, device=DEV)
            ops.gated_delta(both(src), 4, w.to(DEV), taps, row[:, n:n + (taps - 1) * C], both(src), 4 + C + 2,
                            both(low), 3, 3 + H * d, *(x.to(DEV) for x in weights), eps, 1e-6, lay,
                            row[:, :n], H, G, d, dv, out)
            got.append(out[max(1, m - 1):].cpu())
            at += m
        keep = row[slot, n:n + (taps - 1) * C].view(taps - 1, C)
        assert torch.equal(keep.cpu(), raw[T - taps + 1:])
        cache.free_slot(slot)
        cache.free_slot(beside)
        _close(torch.cat(got), ref, 5e-5, f"taps {taps}, {pieces[:4]}")
