"""Bumulix as data: how its configuration maps onto parts, and where its parameters are found in a
weight file.  This is the only file that knows the architecture.

Structure: token embedding (no positions); several residual streams that every sublayer reads
through a weighted sum and writes back to all (hyper-connections), with a root-mean-square norm
whose weight is stored around zero in front of each sublayer and a layer scale behind it; layers
in any order of two mixers, ``attention`` (the difference of two attention maps per head over a
sliding window) and ``latent_attention`` (a cached latent, queries through a latent of their own,
one rotated key part with scaled frequencies, a gate on every number of the heads); a dense
feed-forward (tanh gelu) or none; the sum of the streams, a final norm, the embedding table as
output head, logits bounded by ``c * tanh(z / c)``.  A layer may run with another layer's tensors
and a cache of its own.

Tensor names: ``embed``, ``final.norm``, and per layer ``l<i>.``: ``norm1``, ``norm2``, ``ls1``,
``ls2``, ``hc1.{in, out, mix}``, ``hc2.{in, out, mix}``, ``mix.{q, k, v, o, lq1, lk1, lq2, lk2}`` or
``mix.{dq, dq.norm, uq, dkv, dkv.norm, uk, uv, g, o}``, ``mlp.{up, down}``; every linear weight
stored ``(out, in)``.
"""
from __future__ import annotations

import math

import torch

from ..config.bumulix import BumulixConfig, DifferentialConfig
from ..config.registry import Architecture, register_architecture
from ..engine.spec import LayerSpec, ModelSpec
from ..parts.base import PartSpec
from ..weights.loader import Recipe, Source, WeightPlan, take
from .runesun import _rows


def _owners(cfg: BumulixConfig) -> list[int]:
    """The layers that have tensors of their own, in order."""
    return [i for i, l in enumerate(cfg.layers) if l.weights_of is None]


def _mixer_spec(cfg: BumulixConfig, m) -> PartSpec:
    if isinstance(m, DifferentialConfig):
        return PartSpec("differential_attention", {
            "width": cfg.width, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim,
            "value_dim": m.vdim, "scale": m.scale, "diff": m.diff, "window": m.mask_size,
            "eps": cfg.norm_eps})
    return PartSpec("latent_attention", {
        "width": cfg.width, "n_heads": m.heads, "head_dim": m.dim, "value_dim": m.vdim,
        "latent_dim": m.kv_rank, "scale": m.scale, "eps": cfg.norm_eps, "sink": False, "gate": "each",
        "q_latent_dim": m.q_rank, "rot_dim": m.rot_dim, "rot_dims": m.rot.dims,
        "rot_base": m.rot.base, "rot_scaling": m.rot.scaling()})


def build_spec(cfg: BumulixConfig) -> ModelSpec:
    D = cfg.width
    norm = PartSpec("rmsnorm", {"width": D, "eps": cfg.norm_eps, "zero_centred": True})
    owners = _owners(cfg)
    layers = []
    for i in owners:
        l = cfg.layers[i]
        ffn = None if l.mlp is None else PartSpec("dense_mlp", {
            "width": D, "hidden": l.mlp.ff, "activation": "gelu_tanh", "bias": False})
        layers.append(LayerSpec(
            mixer=_mixer_spec(cfg, l.mixer), ffn=ffn, norm_mixer=norm,
            norm_ffn=None if ffn is None else norm,
            block=PartSpec("hyper_connections", {
                "width": D, "streams": cfg.streams or 1, "residual_mult": cfg.residual_mult,
                "connections": cfg.streams is not None, "ffn": ffn is not None})))
    return ModelSpec(
        architecture="bumulix", vocab_size=cfg.vocab_size, width=D, max_seq_len=None,
        position=PartSpec("none"), layers=tuple(layers), final_norm=norm, tie_head=True,
        schedule=tuple(owners.index(cfg.owner(i)) for i in range(len(cfg.layers))),
        logit_softcap=cfg.logit_softcap, streams=cfg.streams or 1)


def _plain_then_rotated(name: str, heads: int, dim: int, rot: int, width: int) -> Recipe:
    """Query rows stored head after head ``[dim plain | rot rotated]``, held as all heads' plain
    rows, then all heads' rotated rows, then rows of zeros up to a multiple of 8."""
    rows = heads * (dim + rot)

    def combine(ts):
        w = ts[0].view(heads, dim + rot, width)
        parts = [w[:, :dim].reshape(heads * dim, width), w[:, dim:].reshape(heads * rot, width)]
        if rows % 8:
            parts.append(torch.zeros((-rows % 8, width), dtype=w.dtype))
        return torch.cat(parts, dim=0).contiguous()
    return Recipe([Source(name, ((rows, width),))], combine)


def weight_plan(cfg: BumulixConfig, spec: ModelSpec, names: set[str]) -> WeightPlan:
    D, V = cfg.width, cfg.vocab_size
    r: dict[str, Recipe] = {"embedding.table": take("embed", (V, D)),
                            "final_norm.weight": take("final.norm", (D,))}
    ignored = set()
    for n, i in enumerate(_owners(cfg)):
        l = cfg.layers[i]
        m = l.mixer
        p, L = f"l{i}.", f"layers.{n}."
        for q, norm in ((1, "norm_mixer"), (2, "norm_ffn")):
            around = {L + norm + ".weight": (f"{p}norm{q}", (D,)),
                      L + f"block.scale{q}": (f"{p}ls{q}", (D,))}
            if cfg.streams is not None:
                S = cfg.streams
                around.update({L + f"block.in{q}": (f"{p}hc{q}.in", (S,)),
                               L + f"block.out{q}": (f"{p}hc{q}.out", (S,)),
                               L + f"block.mix{q}": (f"{p}hc{q}.mix", (S, S))})
            if q == 2 and l.mlp is None:
                # a layer without feed-forward may still carry what stands around it in the file
                ignored |= {name for name, _ in around.values()}
                continue
            r.update({path: take(name, shape) for path, (name, shape) in around.items()})
        H, d, dv = m.heads, m.dim, m.vdim
        if isinstance(m, DifferentialConfig):
            G = m.kv_heads
            r[L + "mixer.proj.weight"] = _rows([(p + "mix.q", (H * 2 * d, D)), (p + "mix.k", (G * 2 * d, D)),
                                                (p + "mix.v", (G * dv, D))], multiple=8)
            for name in ("lq1", "lk1", "lq2", "lk2"):
                r[L + "mixer." + name] = take(p + "mix." + name, (d,))
        else:
            R, Q, rot = m.kv_rank, m.q_rank, m.rot_dim
            r[L + "mixer.proj.weight"] = _rows([(p + "mix.dq", (Q, D)), (p + "mix.dkv", (R + rot, D)),
                                                (p + "mix.g", (H * dv, D))], multiple=8)
            r[L + "mixer.q_norm"] = take(p + "mix.dq.norm", (Q,))
            r[L + "mixer.q_up.weight"] = _plain_then_rotated(p + "mix.uq", H, d, rot, Q)
            r[L + "mixer.latent_norm"] = take(p + "mix.dkv.norm", (R,))
            # stored [H*d, R]: head i's rows map the latent to its keys; held transposed per head
            r[L + "mixer.key_up"] = Recipe(
                [Source(p + "mix.uk", ((H * d, R),))],
                lambda ts, H=H, d=d, R=R: ts[0].view(H, d, R).transpose(1, 2).contiguous())
            r[L + "mixer.value_up"] = Recipe(
                [Source(p + "mix.uv", ((H * dv, R),))],
                lambda ts, H=H, dv=dv, R=R: ts[0].view(H, dv, R).contiguous())
        r[L + "mixer.out.weight"] = take(p + "mix.o", (D, H * dv))
        if l.mlp is not None:
            r[L + "ffn.fc.weight"] = take(p + "mlp.up", (l.mlp.ff, D))
            r[L + "ffn.proj.weight"] = take(p + "mlp.down", (D, l.mlp.ff))
    return WeightPlan(r, ignored)


def random_tensors(cfg: BumulixConfig, seed: int, *, gain: float = 1.0, std: float | None = None,
                   gamma_jitter: float = 0.1, dtype: torch.dtype = torch.bfloat16) -> dict:
    """Random Bumulix tensors under the names of a weight file.  Matrices ~N(0, gain^2 / in) (or
    ~N(0, std^2) if ``std`` is given), embeddings ~N(0, 1), weights of norms ~N(0, gamma_jitter^2)
    around 0 (the latents' around 1), layer scales 1 + N(0, gamma_jitter^2), streams read in equal
    shares, kept apart and written with 1, each with N(0, gamma_jitter^2) on it; drawn in fp32
    from a seeded CPU generator in a fixed order and stored in ``dtype``."""
    g = torch.Generator(device="cpu")
    g.manual_seed(int(seed))

    def mat(n_out, n_in, s=None):
        s = (gain / math.sqrt(n_in) if std is None else std) if s is None else s
        return (torch.randn(n_out, n_in, generator=g, dtype=torch.float32) * s).to(dtype)

    def vec(n, s, mean=0.0):
        return (torch.randn(n, generator=g, dtype=torch.float32) * s + mean).to(dtype)

    D, V, S = cfg.width, cfg.vocab_size, cfg.streams
    out: dict[str, torch.Tensor] = {"embed": mat(V, D, 1.0)}
    for i in _owners(cfg):
        l = cfg.layers[i]
        m, p = l.mixer, f"l{i}."
        for q in (1, 2) if l.mlp is not None else (1,):
            out[f"{p}norm{q}"] = vec(D, gamma_jitter)
            out[f"{p}ls{q}"] = vec(D, gamma_jitter, 1.0)
            if S is not None:
                out[f"{p}hc{q}.in"] = vec(S, gamma_jitter, 1.0 / S)
                out[f"{p}hc{q}.out"] = vec(S, gamma_jitter, 1.0)
                out[f"{p}hc{q}.mix"] = (torch.eye(S) + torch.randn(S, S, generator=g) * gamma_jitter).to(dtype)
        H, d, dv = m.heads, m.dim, m.vdim
        if isinstance(m, DifferentialConfig):
            out[p + "mix.q"] = mat(H * 2 * d, D)
            out[p + "mix.k"] = mat(m.kv_heads * 2 * d, D)
            out[p + "mix.v"] = mat(m.kv_heads * dv, D)
            for name in ("lq1", "lk1", "lq2", "lk2"):
                out[p + "mix." + name] = vec(d, gamma_jitter)
        else:
            R, Q = m.kv_rank, m.q_rank
            out[p + "mix.dq"] = mat(Q, D)
            out[p + "mix.dq.norm"] = vec(Q, gamma_jitter, 1.0)
            out[p + "mix.uq"] = mat(H * (d + m.rot_dim), Q)
            out[p + "mix.dkv"] = mat(R + m.rot_dim, D)
            out[p + "mix.dkv.norm"] = vec(R, gamma_jitter, 1.0)
            out[p + "mix.uk"] = mat(H * d, R)
            out[p + "mix.uv"] = mat(H * dv, R)
            out[p + "mix.g"] = mat(H * dv, D)
        out[p + "mix.o"] = mat(D, H * dv)
        if l.mlp is not None:
            out[p + "mlp.up"] = mat(l.mlp.ff, D)
            out[p + "mlp.down"] = mat(D, l.mlp.ff)
    out["final.norm"] = vec(D, gamma_jitter)
    return out


ARCHITECTURE = register_architecture(Architecture(
    name="bumulix", config_cls=BumulixConfig, build_spec=build_spec, weight_plan=weight_plan,
    aliases=("Bumulix",), random_tensors=random_tensors), replace=True)
