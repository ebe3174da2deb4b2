"""A plain implementation of the Zorulix decoder: whole sequences, no cache, no batches, one
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


# ----------------------------------------------------------------------------- norms, activations
def over_rms(x, eps):
    """x / sqrt(mean of squares + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def one_plus_norm(x, w, eps):
    """A stored weight of zero leaves the unit row as it is."""
    return over_rms(x, eps) * (1.0 + w)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


# ----------------------------------------------------------------------------- rotation
def pair_rates(dims, base, sc=None):
    """Per pair its angle per position, slow pairs slowed down by ``factor``; the size of cos, sin."""
    rates = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return rates, 1.0

    def place(turns):
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(place(sc["fast"])), 0)
    hi = min(math.ceil(place(sc["slow"])), dims - 1)
    out = []
    for i, f in enumerate(rates):
        t = (i - lo) / max(hi - lo, 0.001)
        t = 0.0 if t < 0 else 1.0 if t > 1 else t
        out.append(f / sc["factor"] * t + f * (1.0 - t))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotated(x, rot):
    """x [T, heads, n], the rows at positions 0 .. T-1: number i of a head with i + dims/2."""
    if not rot:
        return x
    dims = rot["dims"]
    rates, size = pair_rates(dims, rot["base"], rot.get("scaling"))
    T, half = x.shape[0], dims // 2
    ang = torch.arange(T, dtype=torch.float64)[:, None] * torch.tensor(rates, dtype=torch.float64)
    c = (size * torch.cos(ang))[:, None].to(x.dtype)
    s = (size * torch.sin(ang))[:, None].to(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


# ----------------------------------------------------------------------------- attention
def sees(T, size):
    """[T, T] bool: position i (row) sees j with 0 <= i - j < size (no size: every j <= i)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    m = i >= j
    return m & (i - j < size) if size else m


def attend(q, k, v, see, scale, zero_sink):
    """q [T, H, d], k [T, G, d], v [T, G, dv]; ``zero_sink``: one more term exp(0) below the line."""
    T, H = q.shape[:2]
    G = k.shape[1]
    out = q.new_zeros(T, H, v.shape[-1])
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T * scale).masked_fill(~see, -math.inf)
        top = s.max(-1, keepdim=True).values
        if zero_sink:
            top = torch.clamp(top, min=0.0)
        e = torch.exp(s - top)
        below = e.sum(-1, keepdim=True) + (torch.exp(-top) if zero_sink else 0.0)
        out[:, h] = (e / below) @ v[:, g]
    return out


def queries(x, W, p, m, eps, normed):
    q = x @ W[p + "q"].T + W[p + "q.b"]
    if normed:
        q = over_rms(q, eps) * W[p + "q.norm"]       # all heads' numbers at once
    return rotated(q.view(-1, m["heads"], m["dim"]), m.get("rot"))


def keys_values(x, W, p, m, eps, normed):
    k = x @ W[p + "k"].T + W[p + "k.b"]
    if normed:
        k = over_rms(k, eps) * W[p + "k.norm"]
    v = x @ W[p + "v"].T + W[p + "v.b"]
    G = m["kv_heads"]
    return rotated(k.view(-1, G, m["dim"]), m.get("rot")), v.view(-1, G, m["vdim"])


def window_of(m):
    return m["mask"]["size"] if m.get("mask") else 0


def sink_attention(x, W, p, m, eps, store, i):
    """``store``: layer -> its keys and values; a layer with ``kv_from`` reads another's."""
    src = m.get("kv_from")
    if src is None:
        store[i] = keys_values(x, W, p, m, eps, True)
    k, v = store[i if src is None else src]
    o = attend(queries(x, W, p, m, eps, True), k, v, sees(x.shape[0], window_of(m)), m["scale"], True)
    return o.reshape(x.shape[0], -1) @ W[p + "o"].T


def windowed_attention(x, W, p, m, eps):
    k, v = keys_values(x, W, p, m, eps, False)
    o = attend(queries(x, W, p, m, eps, False), k, v, sees(x.shape[0], window_of(m)), m["scale"], False)
    return o.reshape(x.shape[0], -1) @ W[p + "o"].T + W[p + "o.b"]


# ----------------------------------------------------------------------------- the recurrence
def causal_conv(x, w):
    """x [T, C], w [C, taps]: the last tap meets the current token, zeros before the start."""
    taps = w.shape[1]
    padded = torch.cat([x.new_zeros(taps - 1, x.shape[1]), x])
    out = torch.zeros_like(x)
    for j in range(taps):
        out = out + padded[j:j + x.shape[0]] * w[:, j]
    return out


def unit_vectors(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def decays(x, W, p, H, d):
    dt = softplus(x @ W[p + "a1"].T @ W[p + "a2"].T + W[p + "dt_bias"]).view(-1, H, d)
    return torch.exp(-torch.exp(W[p + "A_log"])[:, None] * dt)


def delta_walk(q, k, v, g, beta, S=None):
    """q, k, g [T, H, d], v [T, H, dv], beta [T, H] -> the outputs [T, H, dv] and the last state."""
    T, H, d = q.shape
    dv = v.shape[-1]
    S = q.new_zeros(H, d, dv) if S is None else S.clone()
    out = q.new_zeros(T, H, dv)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return out, S


def gated_delta(x, W, p, m, eps):
    T = x.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(x @ W[p + n].T, W[p + n + ".conv"])) for n in "qkv")
    q = unit_vectors(q.view(T, G, d)) * d ** -0.5
    k = unit_vectors(k.view(T, G, d))
    of = [h // (H // G) for h in range(H)]
    beta = torch.sigmoid(x @ W[p + "b"].T)
    o, _ = delta_walk(q[:, of], k[:, of], v.view(T, H, dv), decays(x, W, p, H, d), beta)
    o = over_rms(o, eps) * W[p + "norm"]
    gate = torch.sigmoid(x @ W[p + "g1"].T @ W[p + "g2"].T)
    return (o.reshape(T, H * dv) * gate) @ W[p + "o"].T


# ----------------------------------------------------------------------------- mixers
def side_by_side(x, W, p, m, eps):
    a = windowed_attention(x, W, p + "left.", m["left"], eps)
    b = gated_delta(x, W, p + "right.", m["right"], eps)
    return m["left_scale"] * a + m["right_scale"] * b


# ----------------------------------------------------------------------------- feed-forward
def expert(x, W, p):
    return (silu(x @ W[p + "gate"].T) * (x @ W[p + "up"].T)) @ W[p + "down"].T


def chosen(z, top):
    """Router logits [T, E] -> the chosen experts [T, top] and the softmax over their logits."""
    val, idx = torch.sort(z, dim=-1, descending=True, stable=True)
    e = torch.exp(val[:, :top] - val[:, :1])
    return idx[:, :top], e / e.sum(-1, keepdim=True)


def router_logits(x, W, p):
    return x @ W[p + "router"].T + W[p + "router.b"]


def experts_mixed(x, W, p, f, choice=None):
    """``choice``: the experts to use instead of the largest logits' (their softmax as it is)."""
    z = router_logits(x, W, p)
    idx, w = chosen(z, f["router"]["top"])
    if choice is not None:
        idx = choice
        w = torch.softmax(torch.gather(z, 1, idx), -1)
    y = torch.zeros_like(x)
    for e in range(z.shape[1]):
        t, k = (idx == e).nonzero(as_tuple=True)
        if len(t):
            y[t] = y[t] + w[t, k][:, None] * expert(x[t], W, f"{p}e{e}.")
    if f.get("shared"):
        y = y + torch.sigmoid(x @ W[p + "shared.sg"].T) * expert(x, W, p + "shared.")
    return y


# ----------------------------------------------------------------------------- token input
def token_input(x, W, p, e, eps):
    y = (gelu_tanh(x @ W[p + "gate"].T) * e) @ W[p + "proj"].T
    return over_rms(y, eps) * W[p + "norm"]


# ----------------------------------------------------------------------------- the model
def layer_forward(x, tokens, W, cfg, i, store, choices=None):
    L, eps, p = cfg["layers"][i], cfg["norm"]["eps"], f"l{i}."
    h = one_plus_norm(x, W[p + "norm1"], eps)
    if L["type"] == "attention":
        x = x + sink_attention(h, W, p + "mix.", L["mixer"], eps, store, i)
    else:
        x = x + side_by_side(h, W, p + "mix.", L["mixer"], eps)
    if L.get("mlp"):
        h = one_plus_norm(x, W[p + "norm2"], eps)
        pick = None if choices is None else choices(i, router_logits(h, W, p + "mlp."))
        x = x + experts_mixed(h, W, p + "mlp.", L["mlp"], pick)
    if cfg.get("token_side"):
        n = cfg["token_side"]["dim"]
        x = x + token_input(x, W, p + "side.", W["side.embed"][tokens][:, i * n:(i + 1) * n], eps)
    return x


def hidden_states(tokens, W, cfg, dtype=torch.float64, choices=None):
    """The stream after every layer, [layers, T, D]."""
    W = widened(W, dtype)
    tokens = torch.tensor(list(tokens))
    x = W["embed"][tokens] * (cfg.get("embedding") or {}).get("scale", 1.0)
    out, store = [], {}
    for i in range(len(cfg["layers"])):
        x = layer_forward(x, tokens, W, cfg, i, store, choices)
        out.append(x)
    return torch.stack(out)


def logits(tokens, W, cfg, dtype=torch.float64, choices=None):
    x = hidden_states(tokens, W, cfg, dtype, choices)[-1]
    W = widened(W, dtype)
    return one_plus_norm(x, W["final.norm"], cfg["norm"]["eps"]) @ W["head"].T
