"""Typed configuration of the Zorulix decoder.

config.json of this design::

    {"architecture": "Zorulix", "vocab": V, "width": D, "norm": {"eps": e},
     "embedding": {"scale": s}, "token_side": {"dim": n},
     "layers": [
       {"type": "attention", "mixer": ATTENTION, "mlp": MLP},
       {"type": "parallel",
        "mixer": {"left": ATTENTION, "left_scale": a,
                  "right": {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "conv": taps},
                  "right_scale": b},
        "mlp": MLP}, ...]}

    ATTENTION = {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": c, "mask": {"size": W},
                 "rot": {"dims": r, "base": b,
                         "scaling": {"factor": f, "original": n, "fast": x, "slow": y}}}
                and, in an "attention" layer only, "kv_from": j
    MLP = {"kind": "moe", "expert": {"ff": F}, "router": {"experts": E, "top": k},
           "shared": {"ff": Fs}} | null

Every size and constant is read from there; layers come in any order and may differ from one
another.  ``attention`` norms all queries and all keys at once and adds one to the softmax's
denominator; a layer with ``kv_from: j`` has queries only and reads the keys and values of layer
``j``, an earlier ``attention`` layer with its own.  ``parallel`` runs a windowed attention and a
gated delta rule beside each other.  Optional keys: ``embedding`` (scale 1), ``token_side`` (none),
``kv_heads`` (= heads), ``vdim`` (= dim), ``scale`` (1 / sqrt(dim)), ``mask`` (every earlier token),
``rot`` and ``rot.scaling`` (none), ``left_scale`` and ``right_scale`` (1), ``shared`` (none).  Two
sizes are not in config.json: the ranks of the delta rule's decay and output gate, which the
weight file's tensor shapes give (``decay_rank``, ``gate_rank``; a config written by this library
carries them).
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Any

from .base import ConfigError
from .runesun import _float, _int

MIXER_TYPES = ("attention", "parallel")


@dataclass(frozen=True)
class RotaryConfig:
    dims: int
    base: float
    factor: float | None = None        # None: no frequency scaling
    original: float = 0.0
    fast: float = 0.0
    slow: float = 0.0

    def scaling(self) -> dict | None:
        return None if self.factor is None else {
            "factor": self.factor, "original": self.original, "fast": self.fast, "slow": self.slow}


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    mask_size: int = 0                 # 0: every earlier token is seen
    rot: RotaryConfig | None = None
    kv_from: int | None = None


@dataclass(frozen=True)
class DeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    decay_rank: int | None = None      # from the weight file's shapes when config.json has none
    gate_rank: int | None = None


@dataclass(frozen=True)
class ParallelConfig:
    left: AttentionConfig
    right: DeltaConfig
    left_scale: float = 1.0
    right_scale: float = 1.0


@dataclass(frozen=True)
class MoEFFConfig:
    experts: int
    top: int
    ff: int
    shared_ff: int | None = None


@dataclass(frozen=True)
class ZorulixLayerConfig:
    type: str
    mixer: Any                         # AttentionConfig or ParallelConfig
    mlp: MoEFFConfig | None


def _has(obj, key) -> bool:
    return isinstance(obj, dict) and obj.get(key) is not None


def _read_heads(problems, where, m) -> tuple[int, int, int, int]:
    heads = _int(problems, where, m, "heads")
    kv_heads = _int(problems, where, m, "kv_heads") if _has(m, "kv_heads") else heads
    dim = _int(problems, where, m, "dim")
    vdim = _int(problems, where, m, "vdim") if _has(m, "vdim") else dim
    if heads % kv_heads:
        problems.append(f"{where}: heads={heads} is no multiple of kv_heads={kv_heads}")
    return heads, kv_heads, dim, vdim


def _read_rot(problems, where, r, dim) -> RotaryConfig:
    dims = _int(problems, where, r, "dims", minimum=2)
    if dims % 2 or dims > dim:
        problems.append(f"{where}.dims: {dims} must be even and at most the head's {dim}")
    rot = RotaryConfig(dims, _float(problems, where, r, "base"))
    if _has(r, "scaling"):
        s = r["scaling"]
        rot = replace(rot, **{k: _float(problems, where + ".scaling", s, k)
                              for k in ("factor", "original", "fast", "slow")})
    return rot


def _read_attention(problems, where, m, layer: int | None) -> AttentionConfig:
    """``layer``: the layer's number where ``kv_from`` may stand, else ``None``."""
    heads, kv_heads, dim, vdim = _read_heads(problems, where, m)
    scale = _float(problems, where, m, "scale", positive=False) if _has(m, "scale") else dim ** -0.5
    size = _int(problems, where + ".mask", m["mask"], "size") if _has(m, "mask") else 0
    rot = _read_rot(problems, where + ".rot", m["rot"], dim) if _has(m, "rot") else None
    src = None
    if _has(m, "kv_from"):
        src = m["kv_from"]
        if layer is None:
            problems.append(f"{where}.kv_from: only an attention layer reads another's keys")
            src = None
        elif isinstance(src, bool) or not isinstance(src, int) or not 0 <= src < layer:
            problems.append(f"{where}.kv_from: {src!r} is not an earlier layer")
            src = None
    return AttentionConfig(heads, kv_heads, dim, vdim, scale, size, rot, src)


def _read_parallel(problems, where, m) -> ParallelConfig:
    left, right = (m.get(k) if isinstance(m, dict) else None for k in ("left", "right"))
    heads, kv_heads, dim, vdim = _read_heads(problems, where + ".right", right)
    ranks = {k: _int(problems, where + ".right", right, k) if _has(right, k) else None
             for k in ("decay_rank", "gate_rank")}
    scales = {k: _float(problems, where, m, k, positive=False) if _has(m, k) else 1.0
              for k in ("left_scale", "right_scale")}
    return ParallelConfig(
        left=_read_attention(problems, where + ".left", left, None),
        right=DeltaConfig(heads, kv_heads, dim, vdim,
                          _int(problems, where + ".right", right, "conv"), **ranks), **scales)


def _read_mlp(problems, where, f) -> MoEFFConfig | None:
    if f is None:
        return None
    if not isinstance(f, dict) or f.get("kind") != "moe":
        problems.append(f"{where}.kind: unknown feed-forward "
                        f"{f.get('kind') if isinstance(f, dict) else f!r} (known: moe, or null)")
        return None
    experts = _int(problems, where + ".router", f.get("router"), "experts")
    top = _int(problems, where + ".router", f.get("router"), "top")
    if top > experts:
        problems.append(f"{where}.router: top={top} of {experts} experts")
    return MoEFFConfig(experts, top, _int(problems, where + ".expert", f.get("expert"), "ff"),
                       _int(problems, where + ".shared", f["shared"], "ff") if _has(f, "shared") else None)


@dataclass(frozen=True)
class ZorulixConfig:
    architecture = "zorulix"

    vocab_size: int
    width: int
    norm_eps: float
    embedding_scale: float
    side_dim: int                      # 0: no per-layer token input
    layers: tuple[ZorulixLayerConfig, ...]
    name: str = "model"

    @classmethod
    def from_json(cls, obj: dict) -> "ZorulixConfig":
        if not isinstance(obj, dict):
            raise ConfigError("config.json must hold a JSON object")
        problems: list[str] = []
        vocab = _int(problems, "config", obj, "vocab")
        width = _int(problems, "config", obj, "width")
        eps = _float(problems, "norm", obj.get("norm"), "eps")
        emb = obj.get("embedding")
        scale = _float(problems, "embedding", emb, "scale", positive=False) if _has(emb, "scale") else 1.0
        side = _int(problems, "token_side", obj["token_side"], "dim") if _has(obj, "token_side") else 0
        raw_layers = obj.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("bad config.json: layers: expected a non-empty list"
                              + ("; " + "; ".join(problems) if problems else ""))
        layers = []
        for i, entry in enumerate(raw_layers):
            where = f"layers[{i}]"
            if not isinstance(entry, dict):
                problems.append(f"{where}: expected an object")
                continue
            kind = entry.get("type")
            if kind not in MIXER_TYPES:
                problems.append(f"{where}.type: unknown mixer {kind!r} (known: {list(MIXER_TYPES)})")
                continue
            m = entry.get("mixer")
            mixer = _read_attention(problems, where + ".mixer", m, i) if kind == "attention" \
                else _read_parallel(problems, where + ".mixer", m)
            layers.append(ZorulixLayerConfig(kind, mixer, _read_mlp(problems, where + ".mlp",
                                                                    entry.get("mlp"))))
        if problems:
            raise ConfigError("bad config.json: " + "; ".join(problems))
        for i, l in enumerate(layers):
            src = l.mixer.kv_from if l.type == "attention" else None
            if src is None:
                continue
            o, m = layers[src], l.mixer
            if o.type != "attention" or o.mixer.kv_from is not None:
                problems.append(f"layers[{i}].mixer.kv_from: layer {src} has no keys and values of its own")
            elif (o.mixer.kv_heads, o.mixer.dim, o.mixer.vdim) != (m.kv_heads, m.dim, m.vdim):
                problems.append(f"layers[{i}].mixer.kv_from: layer {src} keeps "
                                f"{o.mixer.kv_heads} heads of {o.mixer.dim}/{o.mixer.vdim}, not "
                                f"{m.kv_heads} of {m.dim}/{m.vdim}")
        if problems:
            raise ConfigError("bad config.json: " + "; ".join(problems))
        return cls(vocab_size=vocab, width=width, norm_eps=eps, embedding_scale=scale, side_dim=side,
                   layers=tuple(layers), name=str(obj.get("name", "model")))

    def with_shapes(self, shapes: dict) -> "ZorulixConfig":
        """The sizes that only the weight file knows, read off its tensor shapes
        (``{name: shape}``): the ranks of every delta rule's decay and output gate."""
        layers = []
        for i, l in enumerate(self.layers):
            if l.type == "parallel":
                found = {}
                for key, name in (("decay_rank", "a1"), ("gate_rank", "g1")):
                    shape = shapes.get(f"l{i}.mix.right.{name}")
                    if getattr(l.mixer.right, key) is None and shape is not None and len(shape) == 2:
                        found[key] = int(shape[0])
                l = replace(l, mixer=replace(l.mixer, right=replace(l.mixer.right, **found)))
            layers.append(l)
        return replace(self, layers=tuple(layers))

    def n_params(self, *_unused) -> int:
        D, V, n = self.width, self.vocab_size, self.side_dim
        total = 2 * V * D + D + V * n * len(self.layers)

        def attention(m: AttentionConfig, normed: bool) -> int:
            q, k, v = m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim
            rows = q + (k + v if m.kv_from is None else 0)
            norms = (q + (k if m.kv_from is None else 0)) if normed else 0
            return rows * (D + 1) + norms + m.heads * m.vdim * D

        for l in self.layers:
            total += D + (2 * n * D + D if n else 0)
            if l.type == "attention":
                total += attention(l.mixer, True)
            else:
                r = l.mixer.right
                qk, hd, hv = r.kv_heads * r.dim, r.heads * r.dim, r.heads * r.vdim
                ra, rg = r.decay_rank or 0, r.gate_rank or 0
                total += attention(l.mixer.left, False) + D
                total += (2 * qk + hv) * (D + r.taps) + r.heads * (D + 1) + hd + r.vdim + hv * D
                total += (ra + rg) * D + hd * ra + hv * rg
            if l.mlp is not None:
                f = l.mlp
                total += D + f.experts * (3 * f.ff * D + D + 1)
                total += 3 * f.shared_ff * D + D if f.shared_ff is not None else 0
        return total

    def to_json(self) -> dict[str, Any]:
        def attention(m: AttentionConfig) -> dict:
            out: dict[str, Any] = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim,
                                   "vdim": m.vdim, "scale": m.scale}
            if m.mask_size:
                out["mask"] = {"size": m.mask_size}
            if m.rot is not None:
                out["rot"] = {"dims": m.rot.dims, "base": m.rot.base}
                if m.rot.factor is not None:
                    out["rot"]["scaling"] = m.rot.scaling()
            if m.kv_from is not None:
                out["kv_from"] = m.kv_from
            return out

        layers = []
        for l in self.layers:
            if l.type == "attention":
                mx = attention(l.mixer)
            else:
                r = l.mixer.right
                right: dict[str, Any] = {"heads": r.heads, "kv_heads": r.kv_heads, "dim": r.dim,
                                         "vdim": r.vdim, "conv": r.taps}
                for key in ("decay_rank", "gate_rank"):
                    if getattr(r, key) is not None:
                        right[key] = getattr(r, key)
                mx = {"left": attention(l.mixer.left), "left_scale": l.mixer.left_scale,
                      "right": right, "right_scale": l.mixer.right_scale}
            ff = None
            if l.mlp is not None:
                ff = {"kind": "moe", "expert": {"ff": l.mlp.ff},
                      "router": {"experts": l.mlp.experts, "top": l.mlp.top}}
                if l.mlp.shared_ff is not None:
                    ff["shared"] = {"ff": l.mlp.shared_ff}
            layers.append({"type": l.type, "mixer": mx, "mlp": ff})
        obj: dict[str, Any] = {"architecture": "Zorulix", "name": self.name, "vocab": self.vocab_size,
                               "width": self.width, "norm": {"eps": self.norm_eps},
                               "embedding": {"scale": self.embedding_scale}, "layers": layers}
        if self.side_dim:
            obj["token_side"] = {"dim": self.side_dim}
        return obj
