"""Interfaces of the parts a model is assembled from, and their registries.

A *part* is built from a :class:`PartSpec` (a kind name plus keyword arguments: all of
its sizes and constants) and knows nothing about the model it sits in.  There are six
families, each with its own registry:

=============  ===========================================================================
family         interface
=============  ===========================================================================
``norm``       ``forward(ctx, x_f32[rows, width], rows=None) -> act[rows', width]``
``position``   ``table`` (rows added to the token embedding, or ``None``) and
               ``rotate(ctx, qkv)`` (applied to queries and keys before they are cached)
``mixer``      ``forward(ctx, h, residual)``: mixes tokens of a sequence; ``residual`` (the
               fp32 stream) receives ``+= mixer(h)``.  Declares what it keeps per sequence
               with ``cache_request()`` (growing keys/values) and ``state_request()``
               (fixed size); the storage of the running schedule entry is on the context
               (``ctx.kv``, ``ctx.state``, ``ctx.writes_cache``).
``ffn``        ``forward(ctx, h, residual)``: per-token feed-forward, ``residual += ffn(h)``
``block``      ``forward(ctx, x, layer)``: the arrangement of norms, mixer and feed-forward
               around the residual stream of one layer (``layer.ffn`` and ``layer.norm_ffn``
               are ``None`` in a layer without them)
``side``       ``forward(ctx, x, x_act, then=None)``: a per-token input that a layer adds to
               the stream after its sublayers (``x_act``: the stream's rows in the activation
               type; ``then``: a norm whose rows of the new stream are returned)
``stream``     ``forward(ctx, x, x0) -> x'``: acts on the stream right before a schedule entry
               (``x0``: the embedding's output); the model lists which entries
``embedding``  ``forward(ctx, position) -> x``: the fp32 stream from the step's tokens; the
               default is the token table (plus a position table); may keep a state row per
               sequence (``state_request()``, ``ctx.state`` while it runs)
=============  ===========================================================================

Every part lists its parameters with :meth:`Part.param_specs` (shape and role) and gets the
loaded device tensors through :meth:`Part.bind`.
"""
from __future__ import annotations

from dataclasses import dataclass, field, replace
from typing import Any, Callable

import torch

MATRIX = "matrix"   # linear weight held as [out, in]; element type follows the run precision
TABLE = "table"     # rows gathered by index (embeddings); element type as for matrices
VECTOR = "vector"   # biases and norm weights; always held in fp32
INDEX = "index"     # integer tables; held as int32


@dataclass(frozen=True)
class ParamSpec:
    shape: tuple[int, ...]
    role: str = MATRIX
    optional: bool = False


@dataclass(frozen=True)
class PartSpec:
    """Which part, with which sizes and constants."""
    kind: str
    args: dict = field(default_factory=dict)

    def with_args(self, **kw) -> "PartSpec":
        return PartSpec(self.kind, {**self.args, **kw})


@dataclass(frozen=True)
class KVRequest:
    """Growing per-sequence storage a mixer needs: keys and values for every cached token.
    ``window`` > 0 means only the last ``window`` tokens are ever read.  ``planes``: 2 for keys
    and values, 1 for a mixer that keeps one vector per token and head (a latent that is key
    and value at once).  ``every`` > 1: one entry per ``every`` tokens of the sequence instead of
    one per token (a store of pooled blocks: entry ``b`` belongs to tokens ``b * every ..
    b * every + every - 1`` and exists once the last of them is cached).  ``keep_first`` (with a
    window): the sequence's first ``keep_first`` tokens are read by every later token too.
    ``value_dim``: the size of a value where it is not the key's ``head_dim``."""
    n_kv_heads: int
    head_dim: int
    window: int = 0
    planes: int = 2
    every: int = 1
    keep_first: int = 0
    value_dim: int | None = None

    @property
    def value_size(self) -> int:
        return self.head_dim if self.value_dim is None else self.value_dim

    def covering(self, other: "KVRequest") -> "KVRequest":
        """This store kept for a second reader too: nothing that ``other`` sees is given back.
        Both ask for heads and sizes of one kind."""
        if (self.n_kv_heads, self.head_dim, self.value_size, self.planes, self.every) != (
                other.n_kv_heads, other.head_dim, other.value_size, other.planes, other.every):
            raise ValueError(f"one keeps {self}, the other asks for {other}")
        window = max(self.window, other.window) if self.window and other.window else 0
        return replace(self, window=window, keep_first=max(self.keep_first, other.keep_first))


@dataclass(frozen=True)
class StateRequest:
    """Fixed-size per-sequence storage: ``n_elements`` fp32 values, zeroed when a slot is
    handed out."""
    n_elements: int


class Part:
    """Base of all parts."""
    family: str = ""
    kind: str = ""
    #: True if ``forward`` only launches work on the current CUDA stream from device-resident
    #: data (no host reads of the batch, no synchronisation), so that a step can be captured
    #: in a CUDA graph.  A part that does not say so keeps the engine on plain launches.
    graph_safe: bool = False

    def param_specs(self) -> dict[str, ParamSpec]:
        return {}

    def bind(self, params: dict[str, torch.Tensor | None], runtime) -> None:
        """Receive the loaded tensors (``None`` for absent optional ones)."""
        for name, t in params.items():
            setattr(self, name.replace(".", "_"), t)

    def children(self) -> dict[str, "Part"]:
        """Sub-parts whose parameters are listed under ``<name>.``."""
        return {}


class Norm(Part):
    family = "norm"

    def forward(self, ctx, x: torch.Tensor, rows: torch.Tensor | None = None,
                n_rows: int | None = None) -> torch.Tensor:
        raise NotImplementedError

    def defer(self, ctx, x: torch.Tensor):
        """The normalised rows, possibly not computed yet: a consumer that can fuse the norm
        into its first kernel takes a :class:`DeferredNorm` apart, any other calls
        ``.tensor()``.  The default computes right away."""
        return self.forward(ctx, x)


class DeferredNorm:
    """``norm(x)`` that has not been computed: ``x`` fp32 rows, ``args`` what the fused kernel
    needs.  ``tensor()`` computes it the plain way."""

    def __init__(self, ctx, norm: Norm, x: torch.Tensor, args: tuple):
        self.ctx, self.norm, self.x, self.args = ctx, norm, x, args
        self.shape = x.shape
        self.device = x.device

    def tensor(self) -> torch.Tensor:
        return self.norm.forward(self.ctx, self.x)


class Position(Part):
    family = "position"
    #: rows added to the token embedding at a token's position, or None
    table: torch.Tensor | None = None
    #: the longest sequence this encoding can address, or None if unbounded
    max_positions: int | None = None

    def rotate(self, ctx, qkv: torch.Tensor, mixer) -> None:
        """Hook for encodings that act on queries and keys, in place, before keys are written
        to the cache.  ``qkv``: the step's rows [n_rows, q_width + 2 * kv_width] (queries, keys,
        values side by side); ``mixer`` gives ``n_heads``, ``n_kv_heads``, ``head_dim``,
        ``q_width`` and ``kv_width``; a row's position is ``ctx.layout.row_pos``."""
        return None


class Mixer(Part):
    family = "mixer"
    #: True if ``forward`` takes ``h`` as a :class:`DeferredNorm` (its first linear map fuses
    #: the norm); otherwise it always gets a tensor
    accepts_deferred_norm: bool = False

    def cache_request(self) -> KVRequest | None:
        return None

    def state_request(self) -> StateRequest | None:
        return None

    def extra_cache_requests(self) -> tuple[KVRequest, ...]:
        """Further paged stores beside the one of :meth:`cache_request` (pooled blocks, say);
        the running entry's views of them are ``ctx.kv_extra``, in this order."""
        return ()

    def forward(self, ctx, h: torch.Tensor, residual: torch.Tensor) -> None:
        """``ctx.kv``: the paged key/value store of this schedule entry (or of the entry it
        reads from, then ``ctx.writes_cache`` is False); ``ctx.state``: fp32 tensor
        [n_slots, n_elements] or None.  Storage belongs to the schedule entry, not to the
        layer: a layer that runs twice keeps two caches.

        A part that sets ``can_overwrite = True`` also takes ``accumulate=False``: it then
        writes its result over ``residual`` instead of adding to it (an arrangement that norms
        a sublayer's result before the addition hands it a buffer of its own)."""
        raise NotImplementedError


class FeedForward(Part):
    family = "ffn"
    accepts_deferred_norm: bool = False

    def forward(self, ctx, h: torch.Tensor, residual: torch.Tensor) -> None:
        raise NotImplementedError


class Side(Part):
    family = "side"

    def forward(self, ctx, x: torch.Tensor, x_act: torch.Tensor, then: "Norm | None" = None):
        raise NotImplementedError


class Block(Part):
    family = "block"

    def forward(self, ctx, x: torch.Tensor, layer) -> None:
        raise NotImplementedError


_REGISTRIES: dict[str, dict[str, Callable[..., Part]]] = {
    "norm": {}, "position": {}, "mixer": {}, "ffn": {}, "block": {}, "side": {}, "stream": {},
    "embedding": {},
}


def register_part(family: str, kind: str, factory: Callable[..., Part] | None = None, *,
                  replace: bool = False):
    """Register ``factory(**args) -> Part`` under ``family``/``kind``.  Usable as a decorator
    on a class: ``@register_part("mixer", "my_mixer")``."""
    if family not in _REGISTRIES:
        raise ValueError(f"unknown part family {family!r} (have {sorted(_REGISTRIES)})")

    def _do(f):
        if kind in _REGISTRIES[family] and not replace:
            raise ValueError(f"{family} part {kind!r} is already registered")
        _REGISTRIES[family][kind] = f
        if isinstance(f, type):
            f.kind = kind
        return f

    return _do(factory) if factory is not None else _do


def build_part(family: str, spec: PartSpec) -> Part:
    try:
        factory = _REGISTRIES[family][spec.kind]
    except KeyError:
        raise ValueError(
            f"no {family} part named {spec.kind!r} (registered: {sorted(_REGISTRIES[family])})"
        ) from None
    part = factory(**spec.args)
    if not part.kind:
        part.kind = spec.kind
    return part


def registered_parts(family: str) -> list[str]:
    return sorted(_REGISTRIES[family])


def collect_param_specs(part: Part, prefix: str = "") -> dict[str, ParamSpec]:
    """All parameters of a part and its children, keyed by dotted path."""
    out = {prefix + n: s for n, s in part.param_specs().items()}
    for cname, child in part.children().items():
        out.update(collect_param_specs(child, f"{prefix}{cname}."))
    return out


def bind_params(part: Part, params: dict[str, Any], runtime, prefix: str = "") -> None:
    own = {n: params.get(prefix + n) for n in part.param_specs()}
    part.bind(own, runtime)
    for cname, child in part.children().items():
        bind_params(child, params, runtime, f"{prefix}{cname}.")
