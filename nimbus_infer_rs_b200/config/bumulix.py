"""Typed configuration of the Bumulix decoder.

config.json of this design::

    {"architecture": "Bumulix", "vocab": V, "width": D, "norm": {"eps": e},
     "streams": S, "residual_mult": m, "logit_softcap": c,
     "layers": [
       {"type": "attention",
        "mixer": {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": s, "diff": f,
                  "mask": {"size": W}},
        "mlp": {"kind": "dense", "ff": F} | null,
        "weights_of": j (optional)},
       {"type": "latent_attention",
        "mixer": {"heads": H, "dim": d, "rot_dim": r, "vdim": dv, "kv_rank": R, "q_rank": Q,
                  "scale": s,
                  "rot": {"dims": r, "base": b,
                          "scaling": {"factor": f, "original": n, "fast": u, "slow": w}}},
        "mlp": ...}, ...]}

Every size and constant is read from there; layers come in any order and may differ from one
another.  ``attention`` is the difference of two attention maps per head over a sliding window;
``latent_attention`` attends over a cached latent and one rotated key part.  Optional keys:
``kv_heads`` (= heads), ``vdim`` (= dim of the unrotated part; for ``attention`` 2 dim), ``mask``
(every earlier token), ``rot.dims`` (= rot_dim), ``rot.scaling`` (none), ``streams`` (no
connections between streams: one ordinary residual), ``residual_mult`` (1), ``logit_softcap``
(none).  A layer with ``weights_of: j`` has no tensors of its own and runs with layer ``j``'s (its
own cache) and must be described as that layer is.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any

from .base import ConfigError
from .runesun import _float, _int

MIXER_TYPES = ("attention", "latent_attention")
MLP_KINDS = ("dense",)
MAX_STREAMS = 8


@dataclass(frozen=True)
class DifferentialConfig:
    heads: int
    kv_heads: int
    dim: int                     # of one map
    vdim: int
    scale: float
    diff: float
    mask_size: int = 0           # 0: every earlier token is seen


@dataclass(frozen=True)
class ScaledRotaryConfig:
    dims: int
    base: float
    factor: float | None = None  # None: frequencies as they are
    original: float = 0.0
    fast: float = 0.0
    slow: float = 0.0

    def scaling(self) -> dict | None:
        if self.factor is None:
            return None
        return {"factor": self.factor, "original": self.original, "fast": self.fast, "slow": self.slow}


@dataclass(frozen=True)
class RotatedLatentConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rot: ScaledRotaryConfig


@dataclass(frozen=True)
class DenseConfig:
    ff: int


@dataclass(frozen=True)
class BumulixLayerConfig:
    type: str
    mixer: Any                   # DifferentialConfig or RotatedLatentConfig
    mlp: DenseConfig | None
    weights_of: int | None = None


def _has(obj, key) -> bool:
    return isinstance(obj, dict) and obj.get(key) is not None


def _number(v):
    """A float that is a whole number is written back as one."""
    return int(v) if float(v) == int(v) else v


def _read_differential(problems, where, m) -> DifferentialConfig:
    heads = _int(problems, where, m, "heads")
    kv_heads = _int(problems, where, m, "kv_heads") if _has(m, "kv_heads") else heads
    dim = _int(problems, where, m, "dim")
    vdim = _int(problems, where, m, "vdim") if _has(m, "vdim") else 2 * dim
    if heads % kv_heads:
        problems.append(f"{where}: heads={heads} is no multiple of kv_heads={kv_heads}")
    size = _int(problems, where + ".mask", m["mask"], "size") if _has(m, "mask") else 0
    return DifferentialConfig(heads, kv_heads, dim, vdim,
                              _float(problems, where, m, "scale", positive=False),
                              _float(problems, where, m, "diff", positive=False), size)


def _read_rotary(problems, where, r, rot_dim) -> ScaledRotaryConfig:
    dims = _int(problems, where, r, "dims", minimum=2) if _has(r, "dims") else rot_dim
    if dims % 2 or dims > rot_dim:
        problems.append(f"{where}.dims: {dims} must be even and at most rot_dim={rot_dim}")
    base = _float(problems, where, r, "base")
    if not _has(r, "scaling"):
        return ScaledRotaryConfig(dims, base)
    s, at = r["scaling"], where + ".scaling"
    return ScaledRotaryConfig(dims, base, *(_float(problems, at, s, k)
                                            for k in ("factor", "original", "fast", "slow")))


def _read_latent(problems, where, m) -> RotatedLatentConfig:
    dim = _int(problems, where, m, "dim")
    rot_dim = _int(problems, where, m, "rot_dim", minimum=2)
    return RotatedLatentConfig(
        heads=_int(problems, where, m, "heads"), dim=dim, rot_dim=rot_dim,
        vdim=_int(problems, where, m, "vdim") if _has(m, "vdim") else dim,
        kv_rank=_int(problems, where, m, "kv_rank"), q_rank=_int(problems, where, m, "q_rank"),
        scale=_float(problems, where, m, "scale", positive=False),
        rot=_read_rotary(problems, where + ".rot", m.get("rot") if isinstance(m, dict) else None,
                         rot_dim))


@dataclass(frozen=True)
class BumulixConfig:
    architecture = "bumulix"

    vocab_size: int
    width: int
    norm_eps: float
    streams: int | None           # None: one residual without connections
    residual_mult: float
    logit_softcap: float          # 0: logits are not bounded
    layers: tuple[BumulixLayerConfig, ...]
    name: str = "model"

    @classmethod
    def from_json(cls, obj: dict) -> "BumulixConfig":
        if not isinstance(obj, dict):
            raise ConfigError("config.json must hold a JSON object")
        problems: list[str] = []
        vocab = _int(problems, "config", obj, "vocab")
        width = _int(problems, "config", obj, "width")
        eps = _float(problems, "norm", obj.get("norm"), "eps")
        streams = _int(problems, "config", obj, "streams") if _has(obj, "streams") else None
        if streams is not None and streams > MAX_STREAMS:
            problems.append(f"config.streams: at most {MAX_STREAMS} (got {streams})")
        mult = _float(problems, "config", obj, "residual_mult", positive=False) \
            if _has(obj, "residual_mult") else 1.0
        cap = _float(problems, "config", obj, "logit_softcap") if _has(obj, "logit_softcap") else 0.0
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
            read = _read_differential if kind == "attention" else _read_latent
            mixer = read(problems, where + ".mixer", entry.get("mixer"))
            mlp, f = None, entry.get("mlp")
            if f is not None:
                if not isinstance(f, dict) or f.get("kind") not in MLP_KINDS:
                    problems.append(f"{where}.mlp.kind: unknown feed-forward "
                                    f"{f.get('kind') if isinstance(f, dict) else f!r} "
                                    f"(known: {list(MLP_KINDS)}, or null)")
                else:
                    mlp = DenseConfig(_int(problems, where + ".mlp", f, "ff"))
            wo = entry.get("weights_of")
            if wo is not None and (isinstance(wo, bool) or not isinstance(wo, int)
                                   or not 0 <= wo < len(raw_layers) or wo == i):
                problems.append(f"{where}.weights_of: {wo!r} is not another layer")
                wo = None
            layers.append(BumulixLayerConfig(kind, mixer, mlp, wo))
        if problems:
            raise ConfigError("bad config.json: " + "; ".join(problems))
        cfg = cls(vocab_size=vocab, width=width, norm_eps=eps, streams=streams, residual_mult=mult,
                  logit_softcap=cap, layers=tuple(layers), name=str(obj.get("name", "model")))
        for i, l in enumerate(layers):
            j = cfg.owner(i)              # a chain that never reaches tensors fails here
            o = layers[j]
            if j != i and (o.type, o.mixer, o.mlp) != (l.type, l.mixer, l.mlp):
                raise ConfigError(f"bad config.json: layers[{i}] runs with the tensors of layer {j} "
                                  "but is described differently")
        return cfg

    def owner(self, i: int) -> int:
        """The layer whose tensors layer ``i`` runs with (``i`` itself if it has its own)."""
        seen = set()
        while self.layers[i].weights_of is not None:
            if i in seen:
                raise ConfigError(f"bad config.json: layers[{i}].weights_of goes round in a circle")
            seen.add(i)
            i = self.layers[i].weights_of
        return i

    def n_params(self, *_unused) -> int:
        """Parameters of the layers that have tensors of their own, and the (tied) embedding."""
        D, S = self.width, self.streams
        total = self.vocab_size * D + D
        around = 2 * D + (0 if S is None else 2 * S + S * S)     # a sublayer's norm, scale, streams
        for l in self.layers:
            if l.weights_of is not None:
                continue
            m = l.mixer
            total += around * (1 if l.mlp is None else 2)
            if isinstance(m, DifferentialConfig):
                total += D * (2 * m.dim * (m.heads + m.kv_heads) + m.kv_heads * m.vdim
                              + m.heads * m.vdim) + 4 * m.dim
            else:
                total += D * (m.q_rank + m.kv_rank + m.rot_dim + 2 * m.heads * m.vdim) \
                    + m.q_rank * (1 + m.heads * (m.dim + m.rot_dim)) \
                    + m.kv_rank * (1 + m.heads * (m.dim + m.vdim))
            if l.mlp is not None:
                total += 2 * l.mlp.ff * D
        return total

    def to_json(self) -> dict[str, Any]:
        out = []
        for l in self.layers:
            m = l.mixer
            if isinstance(m, DifferentialConfig):
                mx: dict[str, Any] = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim,
                                      "vdim": m.vdim, "scale": m.scale, "diff": m.diff}
                if m.mask_size:
                    mx["mask"] = {"size": m.mask_size}
            else:
                rot: dict[str, Any] = {"dims": m.rot.dims, "base": m.rot.base}
                if m.rot.factor is not None:
                    rot["scaling"] = {**m.rot.scaling(), "original": _number(m.rot.original)}
                mx = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim,
                      "kv_rank": m.kv_rank, "q_rank": m.q_rank, "scale": m.scale, "rot": rot}
            e: dict[str, Any] = {"type": l.type, "mixer": mx,
                                 "mlp": None if l.mlp is None else {"kind": "dense", "ff": l.mlp.ff}}
            if l.weights_of is not None:
                e["weights_of"] = l.weights_of
            out.append(e)
        obj: dict[str, Any] = {"architecture": "Bumulix", "name": self.name, "vocab": self.vocab_size,
                               "width": self.width, "norm": {"eps": self.norm_eps},
                               "residual_mult": self.residual_mult, "layers": out}
        if self.streams is not None:
            obj["streams"] = self.streams
        if self.logit_softcap:
            obj["logit_softcap"] = self.logit_softcap
        return obj
