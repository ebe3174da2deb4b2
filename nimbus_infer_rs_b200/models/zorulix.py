"""Zorulix as data: how its configuration maps onto parts, and where its parameters are found
in a weight file.  This is the only file that knows the architecture.

Structure: token embedding times a constant; pre-norm layers (RMS norms whose stored weight ``w``
means ``1 + w``) in any order of two kinds, ``attention`` (biased projections, all queries and all
keys normed at once, rotated, a sliding window, a sink of score zero; a layer may read another's
keys and values) and ``parallel`` (a windowed attention with scaled rotation frequencies beside a
gated delta rule, their results weighted by two constants); a feed-forward of routed experts
(weights are the softmax over the chosen logits, a shared expert with a gate per token) or none;
after it a per-token input gated by the stream; a final norm and an output head of its own.

Tensor names: ``embed``, ``side.embed`` (all layers' per-token rows side by side), ``final.norm``,
``head``, and per layer ``l<i>.``: ``norm1``, ``norm2``; ``mix.{q, q.b, k, k.b, v, v.b, q.norm,
k.norm, o}``, or ``mix.left.{q, q.b, k, k.b, v, v.b, o, o.b}`` and ``mix.right.{q, k, v, q.conv,
k.conv, v.conv, b, a1, a2, A_log, dt_bias, g1, g2, norm, o}``; ``mlp.{router, router.b, e<k>.{gate,
up, down}, shared.{gate, up, down, sg}}``; ``side.{gate, proj, norm}``; every linear weight stored
``(out, in)``.
"""
from __future__ import annotations

import math

import torch

from ..config.registry import Architecture, register_architecture
from ..config.zorulix import AttentionConfig, DeltaConfig, ZorulixConfig
from ..engine.spec import LayerSpec, ModelSpec
from ..parts.base import PartSpec
from ..weights.loader import Recipe, Source, WeightPlan, take
from .lulizen import _gate_up
from .rizitar import _columns
from .runesun import _rows, _stack

DEFAULT_RANK = 32            # of a model made here without a weight file to give it
UNIT_EPS = 1e-6              # joins the sum of squares of the delta rule's queries and keys


def _ranks(r: DeltaConfig) -> tuple[int, int]:
    return (DEFAULT_RANK if r.decay_rank is None else r.decay_rank,
            DEFAULT_RANK if r.gate_rank is None else r.gate_rank)


def _attention_spec(cfg: ZorulixConfig, m: AttentionConfig, own_layer: bool) -> PartSpec:
    """``own_layer``: the mixer of an ``attention`` layer; else the left one of a pair."""
    return PartSpec("masked_attention", {
        "width": cfg.width, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim,
        "value_dim": m.vdim, "scale": m.scale, "eps": cfg.norm_eps,
        "qk_norm": "whole" if own_layer else False, "window": m.mask_size,
        "sink": "zero" if own_layer else False, "bias": True, "out_bias": not own_layer,
        "rot_dims": 0 if m.rot is None else m.rot.dims,
        "rot_base": 10000.0 if m.rot is None else m.rot.base,
        "rot_scaling": None if m.rot is None else m.rot.scaling(),
        "own_keys": m.kv_from is None})


def build_spec(cfg: ZorulixConfig) -> ModelSpec:
    D = cfg.width
    norm = PartSpec("rmsnorm", {"width": D, "eps": cfg.norm_eps, "zero_centred": True})
    side = None if not cfg.side_dim else PartSpec("gated_token_input", {
        "width": D, "dim": cfg.side_dim, "vocab_size": cfg.vocab_size, "eps": cfg.norm_eps})
    layers = []
    for l in cfg.layers:
        mx, ff = l.mixer, l.mlp
        source = None
        if l.type == "attention":
            mixer, source = _attention_spec(cfg, mx, True), mx.kv_from
        else:
            r = mx.right
            ra, rg = _ranks(r)
            mixer = PartSpec("scaled_pair", {
                "width": D, "left_scale": mx.left_scale, "right_scale": mx.right_scale,
                "left": _attention_spec(cfg, mx.left, False),
                "right": PartSpec("gated_delta_rule", {
                    "width": D, "n_heads": r.heads, "n_kv_heads": r.kv_heads, "head_dim": r.dim,
                    "value_dim": r.vdim, "taps": r.taps, "decay_rank": ra, "gate_rank": rg,
                    "eps": cfg.norm_eps, "key_eps": UNIT_EPS})})
        ffn = None if ff is None else PartSpec("routed_experts", {
            "width": D, "n_experts": ff.experts, "top": ff.top, "hidden": ff.ff,
            "activation": "silu", "renormalize": True, "router_bias": True,
            "shared": None if ff.shared_ff is None else {"hidden": ff.shared_ff, "gate": True}})
        layers.append(LayerSpec(
            mixer=mixer, ffn=ffn, norm_mixer=norm, norm_ffn=None if ffn is None else norm,
            block=PartSpec("pre_norm"), cache_from=source, side=side))
    return ModelSpec(
        architecture="zorulix", vocab_size=cfg.vocab_size, width=D, max_seq_len=None,
        position=PartSpec("none"), layers=tuple(layers), final_norm=norm, tie_head=False,
        embedding_scale=cfg.embedding_scale)


def _vectors(named, multiple: int = 1) -> Recipe:
    """Several vectors end to end, then zeros up to a multiple of ``multiple`` numbers."""
    def combine(ts):
        out = torch.cat([t.to(torch.float32) for t in ts])
        return torch.nn.functional.pad(out, (0, -out.numel() % multiple))
    return Recipe([Source(n, ((size,),)) for n, size in named], combine)


def _attention_plan(r: dict, L: str, p: str, m: AttentionConfig, D: int, own_layer: bool) -> None:
    H, G, d, dv = m.heads, m.kv_heads, m.dim, m.vdim
    named = [("q", H * d)] + ([("k", G * d), ("v", G * dv)] if m.kv_from is None else [])
    r[L + "proj.weight"] = _rows([(p + n, (size, D)) for n, size in named], multiple=8)
    r[L + "proj.bias"] = _vectors([(p + n + ".b", size) for n, size in named], multiple=8)
    r[L + "out.weight"] = take(p + "o", (D, H * dv))
    if own_layer:
        r[L + "q_norm"] = take(p + "q.norm", (H * d,))
        if m.kv_from is None:
            r[L + "k_norm"] = take(p + "k.norm", (G * d,))
    else:
        r[L + "out.bias"] = take(p + "o.b", (D,))


def _delta_plan(r: dict, L: str, p: str, m: DeltaConfig, D: int) -> None:
    H, qk, hd, hv = m.heads, m.kv_heads * m.dim, m.heads * m.dim, m.heads * m.vdim
    (ra, rg), taps = _ranks(m), m.taps
    rank, up = max(ra, rg), max(hd, hv)

    def fill(t, rows):                      # rows of zeros below, up to `rows`
        return torch.nn.functional.pad(t, (0, 0, 0, rows - t.shape[0]))

    def proj(ts):
        if len({t.dtype for t in ts}) > 1:
            ts = [t.to(torch.float32) for t in ts]
        first = torch.cat(ts[:4], dim=0)    # q, k, v, beta; the low-rank maps start on a multiple of 8
        first = fill(first, first.shape[0] + -first.shape[0] % 8)
        out = torch.cat([first, fill(ts[4], rank), fill(ts[5], rank)], dim=0)
        return fill(out, out.shape[0] + -out.shape[0] % 8).contiguous()

    def ups(ts):
        if len({t.dtype for t in ts}) > 1:
            ts = [t.to(torch.float32) for t in ts]
        return torch.stack([torch.nn.functional.pad(t, (0, rank - t.shape[1], 0, up - t.shape[0]))
                            for t in ts]).contiguous()

    r[L + "proj.weight"] = Recipe([Source(p + n, ((size, D),)) for n, size in (
        ("q", qk), ("k", qk), ("v", hv), ("b", H), ("a1", ra), ("g1", rg))], proj)
    r[L + "up"] = Recipe([Source(p + "a2", ((hd, ra),)), Source(p + "g2", ((hv, rg),))], ups)
    r[L + "conv"] = _rows([(p + "q.conv", (qk, taps)), (p + "k.conv", (qk, taps)),
                           (p + "v.conv", (hv, taps))])
    r[L + "a_log"] = take(p + "A_log", (H,))
    r[L + "dt_bias"] = take(p + "dt_bias", (hd,))
    r[L + "norm"] = take(p + "norm", (m.vdim,))
    r[L + "out.weight"] = take(p + "o", (D, hv))


def weight_plan(cfg: ZorulixConfig, spec: ModelSpec, names: set[str]) -> WeightPlan:
    D, V, n_layers = cfg.width, cfg.vocab_size, len(cfg.layers)
    r: dict[str, Recipe] = {"embedding.table": take("embed", (V, D)),
                            "final_norm.weight": take("final.norm", (D,)),
                            "head.weight": take("head", (V, D))}
    ignored = set()
    for i, l in enumerate(cfg.layers):
        p, L = f"l{i}.", f"layers.{i}."
        r[L + "norm_mixer.weight"] = take(p + "norm1", (D,))
        if l.type == "attention":
            _attention_plan(r, L + "mixer.", p + "mix.", l.mixer, D, True)
        else:
            _attention_plan(r, L + "mixer.left.", p + "mix.left.", l.mixer.left, D, False)
            _delta_plan(r, L + "mixer.right.", p + "mix.right.", l.mixer.right, D)
        if l.mlp is None:
            ignored.add(p + "norm2")        # a layer without a feed-forward may still carry its norm
        else:
            E, F, Fs = l.mlp.experts, l.mlp.ff, l.mlp.shared_ff
            r[L + "norm_ffn.weight"] = take(p + "norm2", (D,))
            r[L + "ffn.router_bias"] = take(p + "mlp.router.b", (E,))
            r[L + "ffn.gate"] = _stack([f"{p}mlp.e{k}.gate" for k in range(E)], (F, D))
            r[L + "ffn.up"] = _stack([f"{p}mlp.e{k}.up" for k in range(E)], (F, D))
            r[L + "ffn.down"] = _stack([f"{p}mlp.e{k}.down" for k in range(E)], (D, F))
            if Fs is None:
                r[L + "ffn.router.weight"] = take(p + "mlp.router", (E, D))
            else:
                # the router's rows and the shared expert's gate ride under its two halves
                r[L + "ffn.shared.fc.weight"] = _gate_up(
                    p + "mlp.shared.", Fs, D, extra=[(p + "mlp.router", E), (p + "mlp.shared.sg", 1)])
                r[L + "ffn.shared.proj.weight"] = take(p + "mlp.shared.down", (D, Fs))
        if cfg.side_dim:
            n = cfg.side_dim
            r[L + "side.table"] = _columns("side.embed", (V, n_layers * n), i * n, (i + 1) * n)
            r[L + "side.gate.weight"] = take(p + "side.gate", (n, D))
            r[L + "side.proj.weight"] = take(p + "side.proj", (D, n))
            r[L + "side.norm"] = take(p + "side.norm", (D,))
    return WeightPlan(r, ignored)


def complete_config(cfg: ZorulixConfig, shapes: dict) -> ZorulixConfig:
    return cfg.with_shapes(shapes)


def random_tensors(cfg: ZorulixConfig, seed: int, *, gain: float = 1.0, std: float | None = None,
                   bias_std: float = 0.1, gamma_jitter: float = 0.1,
                   dtype: torch.dtype = torch.bfloat16) -> dict:
    """Random Zorulix tensors under the names of a weight file.  Matrices ~N(0, gain^2 / in) (or
    ~N(0, std^2) if ``std`` is given), embeddings ~N(0, 1) (divided by the embedding's scale, so
    that the stream starts near unit size), plain norm weights 1 + N(0, gamma_jitter^2), those
    stored around zero N(0, gamma_jitter^2), biases ~N(0, bias_std^2); drawn in fp32 from a
    seeded CPU generator in a fixed order and stored in ``dtype``."""
    g = torch.Generator(device="cpu")
    g.manual_seed(int(seed))

    def mat(n_out, n_in, s=None):
        s = (gain / math.sqrt(n_in) if std is None else std) if s is None else s
        return (torch.randn(n_out, n_in, generator=g, dtype=torch.float32) * s).to(dtype)

    def vec(n, s, mean=0.0):
        return (torch.randn(n, generator=g, dtype=torch.float32) * s + mean).to(dtype)

    def attention(p, m: AttentionConfig, own_layer):
        H, G, d, dv = m.heads, m.kv_heads, m.dim, m.vdim
        rows = [("q", H * d)] + ([("k", G * d), ("v", G * dv)] if m.kv_from is None else [])
        for n, size in rows:
            out[p + n] = mat(size, D)
            out[p + n + ".b"] = vec(size, bias_std)
            if own_layer and n != "v":
                out[p + n + ".norm"] = vec(size, gamma_jitter, 1.0)
        out[p + "o"] = mat(D, H * dv)
        if not own_layer:
            out[p + "o.b"] = vec(D, bias_std)

    def delta(p, m: DeltaConfig):
        H, qk, hd, hv = m.heads, m.kv_heads * m.dim, m.heads * m.dim, m.heads * m.vdim
        ra, rg = _ranks(m)
        for n, size in (("q", qk), ("k", qk), ("v", hv)):
            out[p + n] = mat(size, D)
            out[p + n + ".conv"] = mat(size, m.taps, 1.0 / math.sqrt(m.taps))
        out[p + "b"] = mat(H, D)
        out[p + "A_log"] = vec(H, 0.5, -1.0)
        out[p + "dt_bias"] = vec(hd, 0.5, -1.0)
        out[p + "a1"], out[p + "a2"] = mat(ra, D), mat(hd, ra)
        out[p + "g1"], out[p + "g2"] = mat(rg, D), mat(hv, rg)
        out[p + "norm"] = vec(m.vdim, gamma_jitter, 1.0)
        out[p + "o"] = mat(D, hv)

    def expert(p, hidden):
        out[p + "gate"] = mat(hidden, D)
        out[p + "up"] = mat(hidden, D)
        out[p + "down"] = mat(D, hidden)

    D, V, n = cfg.width, cfg.vocab_size, cfg.side_dim
    out: dict[str, torch.Tensor] = {"embed": mat(V, D, 1.0 / max(abs(cfg.embedding_scale), 1e-6))}
    if n:
        out["side.embed"] = mat(V, n * len(cfg.layers), 1.0)
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        out[p + "norm1"] = vec(D, gamma_jitter)
        if l.type == "attention":
            attention(p + "mix.", l.mixer, True)
        else:
            attention(p + "mix.left.", l.mixer.left, False)
            delta(p + "mix.right.", l.mixer.right)
        if l.mlp is not None:
            out[p + "norm2"] = vec(D, gamma_jitter)
            for k in range(l.mlp.experts):
                expert(f"{p}mlp.e{k}.", l.mlp.ff)
            out[p + "mlp.router"] = mat(l.mlp.experts, D)
            out[p + "mlp.router.b"] = vec(l.mlp.experts, bias_std)
            if l.mlp.shared_ff is not None:
                expert(p + "mlp.shared.", l.mlp.shared_ff)
                out[p + "mlp.shared.sg"] = mat(1, D)
        if n:
            out[p + "side.gate"] = mat(n, D)
            out[p + "side.proj"] = mat(D, n)
            out[p + "side.norm"] = vec(D, gamma_jitter, 1.0)
    out["final.norm"] = vec(D, gamma_jitter)
    out["head"] = mat(V, D)
    return out


ARCHITECTURE = register_architecture(Architecture(
    name="zorulix", config_cls=ZorulixConfig, build_spec=build_spec, weight_plan=weight_plan,
    aliases=("Zorulix",), random_tensors=random_tensors, complete_config=complete_config),
    replace=True)
