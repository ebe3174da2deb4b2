"""Two mixers side by side on the same input, their results combined in one pass over the stream."""
from __future__ import annotations

import torch

from .base import VECTOR, Mixer, ParamSpec, PartSpec, StateRequest, build_part, register_part


class MixerPair(Mixer):
    """``left`` and ``right`` (any two mixers, given as part descriptions) read the same rows and
    write into fp32 buffers of their own; ``combine`` (a subclass's) adds the two to the stream
    in one row pass that also hands out, when the arrangement asks for it, the normed rows of the
    stream's next reader.

    Storage: the pair asks for what its branches ask for, the paged stores one after the other
    and the fixed-size state side by side in one row (the left branch's numbers first); each
    branch sees its own part.
    """
    can_overwrite = False
    takes_next_norm = True       # `forward(..., then=norm)` returns that norm's rows of the stream

    def __init__(self, width: int, left: PartSpec, right: PartSpec):
        self.width = int(width)
        self.left = build_part("mixer", left)
        self.right = build_part("mixer", right)
        self.graph_safe = bool(self.left.graph_safe and self.right.graph_safe)
        # paged stores: every branch's own first, then its further ones, in the order asked
        self._stores = []           # (branch index, is_main)
        for b, part in enumerate((self.left, self.right)):
            if part.cache_request() is not None:
                self._stores.append((b, True, part.cache_request()))
            for r in part.extra_cache_requests():
                self._stores.append((b, False, r))
        self._state = [(p.state_request().n_elements if p.state_request() is not None else 0)
                       for p in (self.left, self.right)]

    def children(self):
        return {"left": self.left, "right": self.right}

    def cache_request(self):
        return self._stores[0][2] if self._stores else None

    def extra_cache_requests(self):
        return tuple(s[2] for s in self._stores[1:])

    def state_request(self):
        total = sum(self._state)
        return StateRequest(total) if total else None

    def _branch(self, ctx, b: int, part, h, like):
        """Run one branch on its part of the pair's storage; returns its fp32 result."""
        views = ((ctx.kv,) if self._stores else ()) + tuple(ctx.kv_extra)
        mine = [(v, main) for v, (bb, main, _) in zip(views, self._stores) if bb == b]
        kv, extra, state, writes = ctx.kv, ctx.kv_extra, ctx.state, ctx.writes_cache
        ctx.kv = next((v for v, main in mine if main), None)
        ctx.kv_extra = tuple(v for v, main in mine if not main)
        lo = sum(self._state[:b])
        ctx.state = state[:, lo:lo + self._state[b]] if self._state[b] else None
        try:
            if getattr(part, "can_overwrite", False):
                y = torch.empty_like(like)
                part.forward(ctx, h, y, accumulate=False)
            else:
                y = torch.zeros_like(like)
                part.forward(ctx, h, y)
        finally:
            ctx.kv, ctx.kv_extra, ctx.state, ctx.writes_cache = kv, extra, state, writes
        return y

    def combine(self, ctx, a, b, residual, norm_args) -> None:
        """Add the branches' results to the stream; ``norm_args``: the next reader's norm weight,
        its eps and the rows to fill (or three times nothing)."""
        raise NotImplementedError

    def forward(self, ctx, h: torch.Tensor, residual: torch.Tensor, then=None):
        """``then``: the norm in front of the stream's next reader; its rows are returned."""
        a = self._branch(ctx, 0, self.left, h, residual)
        b = self._branch(ctx, 1, self.right, h, residual)
        nxt = None
        if then is not None:
            nxt = torch.empty(residual.shape, device=residual.device, dtype=ctx.rt.act_dtype)
        self.combine(ctx, a, b, residual, (then.weight, then.eps, nxt) if then is not None
                     else (None, 0.0, None))
        return nxt


@register_part("mixer", "normed_pair")
class NormedPair(MixerPair):
    """Each result is RMS-normed over the width with a weight of its own (``left_norm``,
    ``right_norm``; a plain weight) and the pair's result is ``coef`` times their sum."""

    def __init__(self, width: int, eps: float, left: PartSpec, right: PartSpec, coef: float = 0.5):
        super().__init__(width, left, right)
        self.eps, self.coef = float(eps), float(coef)
        self.left_norm = self.right_norm = None

    def param_specs(self):
        return {"left_norm": ParamSpec((self.width,), VECTOR),
                "right_norm": ParamSpec((self.width,), VECTOR)}

    def combine(self, ctx, a, b, residual, norm_args) -> None:
        ctx.ops.rms_pair_add(a, self.left_norm, b, self.right_norm, self.eps, self.coef, residual,
                             *norm_args)


@register_part("mixer", "scaled_pair")
class ScaledPair(MixerPair):
    """The pair's result is ``left_scale * left + right_scale * right`` (constants)."""

    def __init__(self, width: int, left: PartSpec, right: PartSpec, left_scale: float = 1.0,
                 right_scale: float = 1.0):
        super().__init__(width, left, right)
        self.left_scale, self.right_scale = float(left_scale), float(right_scale)

    def combine(self, ctx, a, b, residual, norm_args) -> None:
        ctx.ops.scaled_pair_add(a, self.left_scale, b, self.right_scale, residual, *norm_args)
