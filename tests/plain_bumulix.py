"""A plain implementation of the Bumulix decoder: whole sequences, no cache, no batches, one
function per mechanism.  It shares no code with the package; the tests compare the engine with it.

Notation: ``T`` tokens, width ``D``; ``W[name]`` are the tensors of a weight file (``l<i>.``
prefixes a layer's); a linear map stored ``[out, in]`` acts as ``x @ W.T``.  Every function works
in the element type of its inputs (float64 in the tests).
"""
from __future__ import annotations

import math

import torch


def widened(tensors: dict, dtype=torch.float64) -> dict:
    return {k: v.to(dtype) if v.is_floating_point() else v for k, v in tensors.items()}


# ----------------------------------------------------------------------------- norms
def unit(x, eps):
    """x / sqrt(mean of squares + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def zero_centred_norm(x, w, eps):
    """A weight of zero leaves the unit row as it is."""
    return unit(x, eps) * (1.0 + w)


def plain_norm(x, w, eps):
    return unit(x, eps) * w


# ----------------------------------------------------------------------------- streams
def read_streams(xs, coef):
    """xs [S, T, D] -> [T, D]: what a sublayer reads (before its norm)."""
    out = torch.zeros_like(xs[0])
    for s in range(xs.shape[0]):
        out = out + coef[s] * xs[s]
    return out


def write_streams(xs, mix, gain, y, m):
    """What the streams become, computed from what they were: stream t is sum_s mix[s, t] xs[s] + m gain[t] y."""
    S = xs.shape[0]
    new = []
    for t in range(S):
        acc = m * gain[t] * y
        for s in range(S):
            acc = acc + mix[s, t] * xs[s]
        new.append(acc)
    return torch.stack(new)


# ----------------------------------------------------------------------------- attention
def weights_over(scores, see):
    """Softmax of [T, T] scores over the places where ``see`` is True."""
    s = scores.masked_fill(~see, -math.inf)
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def sees_window(T, size):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (i - j >= 0) & (i - j < size)


def sees_past(T):
    return torch.arange(T)[:, None] >= torch.arange(T)[None, :]


def map_difference_weight(lq1, lk1, lq2, lk2, diff):
    """What the second map's result is multiplied by before it is taken away from the first's."""
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def difference_of_maps(a1, a2, lam, diff, eps):
    """[..., dv] per head: the difference, brought to unit size, times 1 - diff."""
    return unit(a1 - lam * a2, eps) * (1.0 - diff)


def two_maps(q, k, v, see, scale):
    """q [T, H, 2, d], k [T, G, 2, d], v [T, G, dv] -> both maps' results [T, H, 2, dv]."""
    T, H = q.shape[:2]
    G = k.shape[1]
    out = q.new_zeros(T, H, 2, v.shape[-1])
    for h in range(H):
        g = h // (H // G)
        for a in range(2):
            out[:, h, a] = weights_over(q[:, h, a] @ k[:, g, a].T * scale, see) @ v[:, g]
    return out


def differential_attention(x, W, p, m, eps):
    T = x.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (x @ W[p + "q"].T).view(T, H, 2, d)
    k = (x @ W[p + "k"].T).view(T, G, 2, d)
    v = (x @ W[p + "v"].T).view(T, G, dv)
    see = sees_window(T, m["mask"]["size"]) if m.get("mask") else sees_past(T)
    a = two_maps(q, k, v, see, m["scale"])
    lam = map_difference_weight(*(W[p + n] for n in ("lq1", "lk1", "lq2", "lk2")), m["diff"])
    o = difference_of_maps(a[:, :, 0], a[:, :, 1], lam, m["diff"], eps)
    return o.reshape(T, H * dv) @ W[p + "o"].T


# ----------------------------------------------------------------------------- rotation
def stretched_rates(dims, base, sc):
    """Per pair its angle per position, slow pairs slowed by ``factor``; and the size of cos, sin."""
    rates = []
    for i in range(dims // 2):
        rates.append(base ** (-2.0 * i / dims))
    if not sc:
        return rates, 1.0

    def dim_at(turns):
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(dim_at(sc["fast"])), 0)
    hi = min(math.ceil(dim_at(sc["slow"])), dims - 1)
    for i, f in enumerate(rates):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        rates[i] = f / sc["factor"] * r + f * (1.0 - r)
    return rates, 0.1 * math.log(sc["factor"]) + 1.0


def turned(x, dims, base, sc):
    """x [T, ..., n] with positions 0 .. T-1: number i of the first ``dims`` pairs with i + dims/2."""
    rates, size = stretched_rates(dims, base, sc)
    T, half = x.shape[0], dims // 2
    ang = torch.arange(T, dtype=torch.float64)[:, None] * torch.tensor(rates, dtype=torch.float64)
    shape = (T,) + (1,) * (x.dim() - 2) + (half,)
    c, s = (size * torch.cos(ang)).view(shape).to(x.dtype), (size * torch.sin(ang)).view(shape).to(x.dtype)
    a, b = x[..., :half], x[..., half:dims]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., dims:]], -1)


# ----------------------------------------------------------------------------- latent attention
def latent_attention(x, W, p, m, eps):
    T = x.shape[0]
    H, d, dr, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    rot = m["rot"]
    cq = plain_norm(x @ W[p + "dq"].T, W[p + "dq.norm"], eps)
    q = (cq @ W[p + "uq"].T).view(T, H, d + dr)
    down = x @ W[p + "dkv"].T
    c = plain_norm(down[:, :R], W[p + "dkv.norm"], eps)
    kr = turned(down[:, R:], rot["dims"], rot["base"], rot.get("scaling"))
    k = (c @ W[p + "uk"].T).view(T, H, d)
    v = (c @ W[p + "uv"].T).view(T, H, dv)
    qr = turned(q[..., d:], rot["dims"], rot["base"], rot.get("scaling"))
    out = x.new_zeros(T, H, dv)
    for h in range(H):
        s = (q[:, h, :d] @ k[:, h].T + qr[:, h] @ kr.T) * m["scale"]
        out[:, h] = weights_over(s, sees_past(T)) @ v[:, h]
    out = out.reshape(T, H * dv) * torch.sigmoid(x @ W[p + "g"].T)
    return out @ W[p + "o"].T


# ----------------------------------------------------------------------------- feed-forward
def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def feed_forward(x, W, p):
    return gelu_tanh(x @ W[p + "up"].T) @ W[p + "down"].T


# ----------------------------------------------------------------------------- the model
MIXERS = {"attention": differential_attention, "latent_attention": latent_attention}


def owner(cfg, i):
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def sublayer(xs, W, p, q, f, cfg):
    """Sublayer q (1: mixer, 2: feed-forward) of the layer with prefix p around the function f."""
    eps, m = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
    if cfg.get("streams") is None:                     # an ordinary residual
        return xs + m * W[f"{p}ls{q}"] * f(zero_centred_norm(xs[0], W[f"{p}norm{q}"], eps))
    hc = f"{p}hc{q}."
    y = f(zero_centred_norm(read_streams(xs, W[hc + "in"]), W[f"{p}norm{q}"], eps)) * W[f"{p}ls{q}"]
    return write_streams(xs, W[hc + "mix"], W[hc + "out"], y, m)


def layer_forward(xs, W, cfg, i):
    L, eps = cfg["layers"][i], cfg["norm"]["eps"]
    p = f"l{owner(cfg, i)}."
    xs = sublayer(xs, W, p, 1, lambda h: MIXERS[L["type"]](h, W, p + "mix.", L["mixer"], eps), cfg)
    if L.get("mlp"):
        xs = sublayer(xs, W, p, 2, lambda h: feed_forward(h, W, p + "mlp."), cfg)
    return xs


def hidden_states(tokens, W, cfg, dtype=torch.float64):
    """The sum of the streams after every layer run, [runs, T, D]."""
    W = widened(W, dtype)
    x = W["embed"][torch.tensor(list(tokens))]
    xs = torch.stack([x] * cfg.get("streams", 1))
    out = []
    for i in range(len(cfg["layers"])):
        xs = layer_forward(xs, W, cfg, i)
        out.append(xs.sum(0))
    return torch.stack(out)


def capped(z, cap):
    return cap * torch.tanh(z / cap) if cap else z


def logits(tokens, W, cfg, dtype=torch.float64):
    x = hidden_states(tokens, W, cfg, dtype)[-1]
    W = widened(W, dtype)
    x = zero_centred_norm(x, W["final.norm"], cfg["norm"]["eps"])
    return capped(x @ W["embed"].T, cfg.get("logit_softcap"))
