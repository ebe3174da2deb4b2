"""Small Zorulix configurations with random weights for the tests, made here (own drawing of the
values; the weight file is written by the Runesun tests' own writer) so that the engine reads
them as it reads any model folder and the plain implementation gets the very same numbers as a
dict."""
from __future__ import annotations

import math
from pathlib import Path

import torch

from runesun_models import write_model


def attn(heads, kv_heads, dim, vdim, scale, window=None, rot=None, base=10000.0, scaling=None,
         kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window}
    if rot:
        m["rot"] = {"dims": rot, "base": base}
        if scaling is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def moe(ff, experts, top, shared=None):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def one(mixer, mlp):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def two(left, right, mlp, left_scale=1.0, right_scale=1.0):
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}}


def model(vocab, width, layers, scale=1.0, side=None, eps=1e-5):
    cfg = {"architecture": "Zorulix", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "embedding": {"scale": scale}, "layers": layers}
    if side:
        cfg["token_side"] = {"dim": side}
    return cfg


# A: odd sizes; values of another size than keys; a reader with a longer window than the store's
#    owner, another layer between them; q/k heads shared in the recurrence, more value than key
#    channels; ranks that differ; a layer without feed-forward, one without a shared expert
# B: multiples of 16 (the tensor-core kernels): keys of 32 with values of 64, windows beside a
#    page's length, readers with shorter, equal and longer windows
# C: the smallest of everything: one head of one or two numbers, a window of one token, a
#    convolution of one tap, one expert, no token input, a factor of one on everything
# D: nothing a multiple of 8; no window; a part of the numbers turned; values narrower than keys
# E: heads of 64 and 128; a recurrence of 128 x 64; a reader of a store without a window
CONFIGS = {
    "A": model(211, 56, [
        one(attn(4, 2, 12, 20, 0.4, 9, 12, 500.0), moe(24, 7, 2, 40)),
        two(attn(3, 1, 10, 18, 0.5, 33, 8, 300.0, (4.0, 64, 8.0, 0.5)), delta(4, 2, 9, 13, 4),
            moe(20, 5, 3, 28), 1.4, 0.6),
        one(attn(6, 2, 12, 20, 0.3, 70, 12, 500.0, kv_from=0), None),
        two(attn(2, 2, 6, 14, 0.45, 5, 6, 50.0), delta(3, 1, 6, 10, 2), moe(12, 6, 2), -0.7, 1.3),
        one(attn(2, 2, 12, 20, 0.5, 4, 12, 500.0, kv_from=0), moe(16, 3, 1, 12)),
    ], scale=5.0, side=10, eps=3e-5),
    "B": model(320, 128, [
        one(attn(4, 2, 64, 64, 0.2, 65, 64, 20000.0), moe(64, 8, 2, 64)),
        two(attn(8, 1, 32, 64, 0.25, 128, 32, 10000.0, (8.0, 128, 32.0, 1.0)), delta(4, 4, 32, 32, 4),
            moe(32, 8, 4, 128), 1.1, 0.7),
        one(attn(4, 2, 64, 64, 0.2, 40, 64, 20000.0, kv_from=0), moe(64, 4, 2, 64)),
        one(attn(4, 2, 64, 64, 0.2, 65, 64, 20000.0, kv_from=0), moe(64, 4, 2, 64)),
        two(attn(4, 2, 16, 48, 0.3, 64, 16), delta(4, 2, 64, 48, 3), moe(32, 8, 4, 128), 0.8, 0.9),
        one(attn(8, 2, 64, 64, 0.15, 100, 64, 20000.0, kv_from=0), moe(64, 4, 2, 64)),
    ], scale=8.0, side=16, eps=1e-6),
    "C": model(29, 8, [
        one(attn(1, 1, 2, 1, 1.0, 1, 2, 10.0), moe(3, 1, 1, 2)),
        two(attn(1, 1, 1, 2, 0.7, 3), delta(1, 1, 1, 1, 1), moe(1, 2, 1, 1)),
        one(attn(2, 1, 2, 1, 0.8, 7, 2, 10.0, kv_from=0), None),
    ]),
    "D": model(99, 44, [
        two(attn(5, 5, 10, 6, 0.33, None, 6, 77.0, (2.5, 20, 3.0, 0.7)), delta(5, 5, 11, 9, 3),
            moe(9, 5, 5, 11), 0.9, -1.1),
        one(attn(6, 2, 11, 7, 0.4, 70, 4, 33.0), moe(13, 9, 3, 7)),
        one(attn(4, 2, 11, 7, 0.35, 66, 4, 33.0, kv_from=1), moe(5, 4, 2)),
    ], scale=0.5, side=13),
    "E": model(130, 96, [
        one(attn(2, 1, 128, 128, 0.1, None, 32, 3000.0), moe(40, 6, 2, 24)),
        two(attn(3, 3, 64, 128, 0.12, 130, 64, 10000.0, (16.0, 64, 4.0, 1.0)), delta(2, 1, 128, 64, 4),
            moe(48, 4, 2, 32), 1.0, 1.0),
        one(attn(3, 1, 128, 128, 0.09, 90, 32, 3000.0, kv_from=0), moe(40, 6, 2, 24)),
        two(attn(2, 1, 128, 64, 0.1, 63), delta(2, 2, 48, 130, 4), None, 0.8, 1.2),
    ], scale=3.0, side=32),
}
SEEDS = {"A": 51, "B": 52, "C": 53, "D": 54, "E": 55}
# decay rank, gate rank of the recurrences
RANKS = {"A": (6, 10), "B": (16, 16), "C": (1, 1), "D": (3, 2), "E": (24, 8)}


def make_tensors(cfg: dict, seed: int, ranks=(8, 8)) -> dict[str, torch.Tensor]:
    """fp32 tensors whose values are exact in bfloat16."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, s=1.0, mean=0.0):
        return (torch.randn(*shape, generator=g) * s + mean).to(torch.bfloat16).float()

    def mat(rows, cols, s=1.2):
        return rnd(rows, cols, s=s / math.sqrt(cols))

    D = cfg["width"]
    out = {"embed": rnd(cfg["vocab"], D, s=1.0 / (cfg["embedding"]["scale"]))}

    def attention(p, m, normed):
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n, rows in (("q", H * d), ("k", G * d), ("v", G * dv)):
            if n != "q" and m.get("kv_from") is not None:
                continue
            out[p + n] = mat(rows, D)
            out[p + n + ".b"] = rnd(rows, s=0.3)
            if normed and n != "v":
                out[p + n + ".norm"] = rnd(rows, s=0.3, mean=1.0)
        out[p + "o"] = mat(D, H * dv, 1.0)
        if not normed:
            out[p + "o.b"] = rnd(D, s=0.3)

    def recurrence(p, m):
        H, G, d, dv, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
        for n, rows in (("q", G * d), ("k", G * d), ("v", H * dv)):
            out[p + n] = mat(rows, D)
            out[p + n + ".conv"] = rnd(rows, taps, s=0.5, mean=0.25)
        out[p + "b"] = mat(H, D)
        out[p + "A_log"] = rnd(H, s=0.6, mean=-1.0)
        out[p + "dt_bias"] = rnd(H * d, s=0.6, mean=-1.5)
        out[p + "norm"] = rnd(dv, s=0.2, mean=1.0)
        for a, b, rows, rank in (("a1", "a2", H * d, ranks[0]), ("g1", "g2", H * dv, ranks[1])):
            out[p + a], out[p + b] = mat(rank, D), mat(rows, rank)
        out[p + "o"] = mat(D, H * dv, 1.0)

    def gated(p, hidden):
        out[p + "gate"], out[p + "up"], out[p + "down"] = mat(hidden, D), mat(hidden, D), mat(D, hidden, 1.0)

    n = (cfg.get("token_side") or {}).get("dim")
    if n:
        out["side.embed"] = rnd(cfg["vocab"], n * len(cfg["layers"]))
    for i, l in enumerate(cfg["layers"]):
        m, f, p = l["mixer"], l["mlp"], f"l{i}."
        out[p + "norm1"] = rnd(D, s=0.3)
        if l["type"] == "attention":
            attention(p + "mix.", m, True)
        else:
            attention(p + "mix.left.", m["left"], False)
            recurrence(p + "mix.right.", m["right"])
        if f:
            out[p + "norm2"] = rnd(D, s=0.3)
            for k in range(f["router"]["experts"]):
                gated(f"{p}mlp.e{k}.", f["expert"]["ff"])
            out[p + "mlp.router"] = mat(f["router"]["experts"], D)
            out[p + "mlp.router.b"] = rnd(f["router"]["experts"], s=0.7)
            if f.get("shared"):
                gated(p + "mlp.shared.", f["shared"]["ff"])
                out[p + "mlp.shared.sg"] = mat(1, D)
        if n:
            out[p + "side.gate"], out[p + "side.proj"] = mat(n, D), mat(D, n)
            out[p + "side.norm"] = rnd(D, s=0.3, mean=0.7)
    out["final.norm"] = rnd(D, s=0.3)
    out["head"] = mat(cfg["vocab"], D)
    return out


def make(root: Path, name: str):
    """``(folder, config, tensors)`` of configuration ``name``."""
    cfg = CONFIGS[name]
    tensors = make_tensors(cfg, SEEDS[name], RANKS[name])
    return write_model(Path(root) / f"zorulix_{name}", cfg, tensors), cfg, tensors
