"""Small Bumulix configurations with random weights for the tests, made here (own drawing of the
values; the weight file is written by the Runesun tests' own writer) so that the engine reads
them as it reads any model folder and the plain implementation gets the very same numbers as a
dict."""
from __future__ import annotations

import math
from pathlib import Path

import torch

from runesun_models import write_model


def pair(heads, kv_heads, dim, vdim, scale, diff, window=None):
    """Mixer 'attention': the difference of two maps of ``dim``."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if window is not None:
        m["mask"] = {"size": window}
    return m


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base, scaling=None, dims=None):
    rot = {"dims": rot_dim if dims is None else dims, "base": base}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
            "q_rank": q_rank, "scale": scale, "rot": rot}


def layer(mx, ff, weights_of=None):
    out = {"type": "latent_attention" if "kv_rank" in mx else "attention", "mixer": mx,
           "mlp": None if ff is None else {"kind": "dense", "ff": ff}}
    if weights_of is not None:
        out["weights_of"] = weights_of
    return out


def model(vocab, width, layers, streams=None, mult=None, cap=None, eps=1e-5):
    cfg = {"architecture": "Bumulix", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "layers": layers}
    for key, v in (("streams", streams), ("residual_mult", mult), ("logit_softcap", cap)):
        if v is not None:
            cfg[key] = v
    return cfg


_A1 = latent(3, 14, 10, 12, 20, 18, 0.3, 500.0, (4.0, 64, 8.0, 0.5))
# A: odd sizes; values of another size than two keys (two stores); a window shorter than a page; a
#    layer without feed-forward; layers that run with another's tensors, beside each other and apart
# B: multiples of 16 (the tensor-core kernels): values of twice a map's size over shared key heads,
#    windows beside a page's length, a latent with a rotated part, four streams
# C: the smallest of everything: one stream, one head of one number, a window of one token, no cap,
#    no multiplier, no frequency scaling
# D: nothing a multiple of 8; five streams; values narrower than keys; a part of the rotated numbers
#    turned; a negative share of the second map; no window
# E: no connections between streams: one ordinary residual with layer scales; heads of 128 in a
#    map; a latent longer than a page
CONFIGS = {
    "A": model(211, 56, [
        layer(pair(4, 2, 12, 20, 0.3, 0.4, 9), 40),
        layer(_A1, 52),
        layer(_A1, 52, weights_of=1),
        layer(pair(2, 1, 24, 24, 0.2, 0.7, 40), None),
        layer(pair(4, 2, 12, 20, 0.3, 0.4, 9), 40, weights_of=0),
    ], streams=3, mult=0.7, cap=12.0, eps=3e-5),
    "B": model(320, 128, [
        layer(pair(4, 2, 32, 64, 0.17, 0.5, 100), 256),
        layer(latent(4, 32, 16, 32, 64, 48, 0.14, 10000.0, (8.0, 128, 32.0, 1.0)), 128),
        layer(pair(2, 1, 64, 128, 0.12, 0.8, 64), 128),
        layer(pair(4, 2, 32, 64, 0.17, 0.5, 100), 256, weights_of=0),
        layer(latent(8, 64, 64, 64, 128, 64, 0.09, 100000.0), None),
    ], streams=4, mult=0.4, cap=20.0, eps=1e-6),
    "C": model(29, 8, [
        layer(pair(1, 1, 1, 2, 1.0, 0.3, 1), 3),
        layer(latent(1, 1, 2, 1, 2, 2, 0.7, 10.0), 1),
        layer(pair(2, 1, 3, 6, 0.5, 0.2, 7), None),
    ], streams=1),
    "D": model(99, 44, [
        layer(latent(5, 7, 10, 9, 22, 13, 0.33, 77.0, (2.5, 20, 3.0, 0.7), dims=6), 33),
        layer(pair(6, 2, 10, 6, 0.4, -0.3), 27),
        layer(pair(3, 3, 7, 14, 0.35, 0.9, 70), 21),
    ], streams=5, mult=1.3, cap=5.0),
    "E": model(130, 96, [
        layer(pair(2, 2, 128, 96, 0.08, 0.6, 65), 64),
        layer(latent(2, 48, 32, 80, 72, 40, 0.11, 3000.0, (16.0, 64, 4.0, 1.0)), 64),
        layer(pair(3, 1, 16, 32, 0.25, 0.45), 48),
    ], mult=0.6, cap=9.0),
}
SEEDS = {"A": 41, "B": 42, "C": 43, "D": 44, "E": 45}


def make_tensors(cfg: dict, seed: int) -> dict[str, torch.Tensor]:
    """fp32 tensors whose values are exact in bfloat16."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, s=1.0, mean=0.0):
        return (torch.randn(*shape, generator=g) * s + mean).to(torch.bfloat16).float()

    def mat(rows, cols, s=1.2):
        return rnd(rows, cols, s=s / math.sqrt(cols))

    D, S = cfg["width"], cfg.get("streams")
    out = {"embed": rnd(cfg["vocab"], D)}
    for i, l in enumerate(cfg["layers"]):
        if l.get("weights_of") is not None:
            continue
        m, ff, p = l["mixer"], l["mlp"], f"l{i}."
        for q in (1, 2) if ff else (1,):
            out[f"{p}norm{q}"] = rnd(D, s=0.3)
            out[f"{p}ls{q}"] = rnd(D, s=0.3, mean=1.0)
            if S is not None:
                out[f"{p}hc{q}.in"] = rnd(S, s=0.3, mean=1.0 / S)
                out[f"{p}hc{q}.out"] = rnd(S, s=0.4, mean=1.0)
                out[f"{p}hc{q}.mix"] = (0.6 * torch.eye(S) + rnd(S, S, s=0.3)).to(torch.bfloat16).float()
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        if l["type"] == "attention":
            G = m["kv_heads"]
            for n, rows in (("q", H * 2 * d), ("k", G * 2 * d), ("v", G * dv)):
                out[p + "mix." + n] = mat(rows, D)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                out[p + "mix." + n] = rnd(d, s=0.4 / math.sqrt(d), mean=0.2 / math.sqrt(d))
        else:
            R, Q, r = m["kv_rank"], m["q_rank"], m["rot_dim"]
            for n, rows, cols in (("dq", Q, D), ("uq", H * (d + r), Q), ("dkv", R + r, D),
                                  ("uk", H * d, R), ("uv", H * dv, R), ("g", H * dv, D)):
                out[p + "mix." + n] = mat(rows, cols)
            out[p + "mix.dq.norm"] = rnd(Q, s=0.2, mean=1.0)
            out[p + "mix.dkv.norm"] = rnd(R, s=0.2, mean=1.0)
        out[p + "mix.o"] = mat(D, H * dv, 1.0)
        if ff:
            out[p + "mlp.up"] = mat(ff["ff"], D)
            out[p + "mlp.down"] = mat(D, ff["ff"], 1.0)
    out["final.norm"] = rnd(D, s=0.3)
    return out


def make(root: Path, name: str):
    """``(folder, config, tensors)`` of configuration ``name``."""
    cfg = CONFIGS[name]
    tensors = make_tensors(cfg, SEEDS[name])
    return write_model(Path(root) / f"bumulix_{name}", cfg, tensors), cfg, tensors
