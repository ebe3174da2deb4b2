"""Arrangements of norms, mixer and feed-forward around the residual stream."""
from __future__ import annotations

import torch

from .base import VECTOR, Block, ParamSpec, register_part
from .norm import RMSNorm


@register_part("block", "pre_norm")
class PreNormBlock(Block):
    """``x += mixer(norm_mixer(x)); x += ffn(norm_ffn(x))`` (src/model.rs:297-300 with
    :345-357, :437-439, :448-460, :485-487).  ``x`` is the fp32 residual stream.  The
    feed-forward may be absent.  A mixer that adds its result
    in a row pass of its own (``takes_next_norm``) is given the feed-forward's norm and hands
    back that norm's rows, computed in the same pass.

    A per-token input (``layer.side``) comes last.  It multiplies the stream by a matrix, so it
    wants the stream's rows in the activation type, which a feed-forward whose last kernel is a
    row pass (``hands_out_rounded``) leaves beside its addition; and its own pass over the stream
    also norms it for the layer that runs next (``ctx.next_norm``, ``ctx.normed``)."""
    graph_safe = True
    takes_handed_norm = True

    def __init__(self):
        pass

    def forward(self, ctx, x, layer) -> None:
        mixer, ffn, side = layer.mixer, layer.ffn, layer.side
        h, ctx.normed = ctx.normed, None
        if h is None:
            h = layer.norm_mixer.defer(ctx, x) if mixer.accepts_deferred_norm \
                else layer.norm_mixer.forward(ctx, x)
        rounded = x if side is None or ctx.rt.act_dtype == torch.float32 else None
        if ffn is not None:
            h = self._mix(ctx, h, x, layer)
            if rounded is None and getattr(ffn, "hands_out_rounded", False):
                rounded = torch.empty(x.shape, device=x.device, dtype=ctx.rt.act_dtype)
                ffn.forward(ctx, h, x, rounded=rounded)
            else:
                ffn.forward(ctx, h, x)
        else:
            mixer.forward(ctx, h, x)
        if side is None:
            return
        if rounded is None:
            rounded = torch.empty(x.shape, device=x.device, dtype=ctx.rt.act_dtype)
            ctx.ops.cast_cols(x, rounded, 0)
        then = ctx.next_norm if isinstance(ctx.next_norm, RMSNorm) else None
        ctx.normed = side.forward(ctx, x, rounded, then)

    @staticmethod
    def _mix(ctx, h, x, layer):
        """The mixer's result into the stream; returns the feed-forward's normed rows."""
        mixer, ffn = layer.mixer, layer.ffn
        if getattr(mixer, "takes_next_norm", False) and hasattr(layer.norm_ffn, "add_into"):
            return mixer.forward(ctx, h, x, then=layer.norm_ffn)
        mixer.forward(ctx, h, x)
        return layer.norm_ffn.defer(ctx, x) if ffn.accepts_deferred_norm \
            else layer.norm_ffn.forward(ctx, x)


@register_part("block", "parallel")
class ParallelBlock(Block):
    """``h = norm_mixer(x); x += mixer(h) + ffn(h)``: one norm, both sublayers read its output
    (the feed-forward may be absent).  Each sublayer adds into the fp32 stream; since neither
    reads the stream, the order of the two additions only changes the rounding."""
    graph_safe = True

    def __init__(self):
        pass

    def forward(self, ctx, x, layer) -> None:
        h = layer.norm_mixer.forward(ctx, x)
        layer.mixer.forward(ctx, h, x)
        if layer.ffn is not None:
            layer.ffn.forward(ctx, h, x)


@register_part("block", "sandwich")
class SandwichBlock(Block):
    """A norm before and after each sublayer: ``x += post_norm_mixer(mixer(norm_mixer(x)))``,
    then ``x += post_norm_ffn(ffn(norm_ffn(x)))`` (the feed-forward may be absent), then the
    layer's per-token input if it has one (``layer.side``), which reads the stream itself.

    A sublayer writes its result into an fp32 buffer of its own (a part that cannot overwrite
    gets zeros to add to); one pass over the rows norms that result, adds it to the stream and
    produces what the next reader wants: the next sublayer's normed rows, or the stream rounded
    to the activation type for the per-token input, or (``ctx.next_norm``) the normed rows the
    next layer's mixer reads, which that layer then finds in ``ctx.normed`` and does not compute
    again."""
    graph_safe = True
    takes_handed_norm = True

    def __init__(self):
        pass

    @staticmethod
    def _run(part, ctx, h, like):
        if getattr(part, "can_overwrite", False):
            y = torch.empty_like(like)
            part.forward(ctx, h, y, accumulate=False)
        else:
            y = torch.zeros_like(like)
            part.forward(ctx, h, y)
        return y

    def forward(self, ctx, x, layer) -> None:
        side = layer.side
        # the side input multiplies the stream by a matrix: in a 32-bit run the stream itself
        wants_rounded = side is not None and ctx.rt.act_dtype != torch.float32
        h, ctx.normed = ctx.normed, None
        if h is None:
            h = layer.norm_mixer.forward(ctx, x)
        y = self._run(layer.mixer, ctx, h, x)
        last = layer.post_norm_ffn if layer.ffn is not None else layer.post_norm_mixer
        # the next layer's first norm in the last pass: only if nothing changes the stream after
        # that pass, and the two norms are of one kind (one kernel norms both ways)
        then = ctx.next_norm if side is None and type(ctx.next_norm) is type(last) else None
        if layer.ffn is not None:
            h, _ = layer.post_norm_mixer.add_into(ctx, y, x, then=layer.norm_ffn)
            y = self._run(layer.ffn, ctx, h, x)
        ctx.normed, xr = last.add_into(ctx, y, x, then=then, rounded=wants_rounded)
        if side is not None:
            side.forward(ctx, x, xr if wants_rounded else x)


@register_part("block", "hyper_connections")
class HyperConnectionsBlock(Block):
    """Several residual streams: a sublayer reads a weighted sum of them, and its result is written
    back to all while they are mixed with one another.  For sublayer ``q`` (1 mixer, 2
    feed-forward, which may be absent) of a layer

        ``u = sum_s in_q[s] x_s``;  ``y = ls_q * sublayer(norm(u))``;
        ``x_t <- sum_s mix_q[s, t] x_s + residual_mult * out_q[t] * y``   (all from the old streams)

    ``ls_q`` scales the result number by number (``layer_scale=False``: not).  ``streams=1`` with
    ``connections=False`` is the ordinary residual with a layer scale and a multiplier.

    ``x`` is fp32 ``[rows, streams * width]``, stream after stream.  One pass over a row writes a
    sublayer's result back and hands out what reads the streams next: the normed rows of the
    layer's feed-forward, those of the next layer's mixer (left in ``ctx.normed``), or at the end
    of the model the sum of the streams (``ctx.streams_sum``).  The first write-back of a step
    reads the embedding's single row (``ctx.streams_from``), which all streams equal until then."""
    graph_safe = True
    takes_handed_norm = True

    def __init__(self, width: int, streams: int = 1, residual_mult: float = 1.0,
                 layer_scale: bool = True, connections: bool = True, ffn: bool = True):
        self.width, self.streams = int(width), int(streams)
        self.residual_mult = float(residual_mult)
        self.layer_scale, self.connections = bool(layer_scale), bool(connections)
        if self.streams > 1 and not self.connections:
            raise ValueError("several streams need their connections")
        self.sublayers = (1, 2) if ffn else (1,)
        for q in (1, 2):
            for n in ("in", "out", "mix", "scale", "gain"):
                setattr(self, f"{n}{q}", None)

    def param_specs(self):
        S, specs = self.streams, {}
        for q in self.sublayers:
            if self.connections:
                specs.update({f"in{q}": ParamSpec((S,), VECTOR), f"out{q}": ParamSpec((S,), VECTOR),
                              f"mix{q}": ParamSpec((S, S), VECTOR)})
            if self.layer_scale:
                specs[f"scale{q}"] = ParamSpec((self.width,), VECTOR)
        return specs

    def bind(self, params, runtime) -> None:
        super().bind(params, runtime)
        one = torch.ones(1, dtype=torch.float32, device=runtime.device)
        for q in self.sublayers:
            if not self.connections:
                setattr(self, f"in{q}", one)
                setattr(self, f"out{q}", one)
                setattr(self, f"mix{q}", one.view(1, 1))
            if not self.layer_scale:
                setattr(self, f"scale{q}", torch.ones(self.width, dtype=torch.float32,
                                                      device=runtime.device))
            out = getattr(self, f"out{q}")
            setattr(self, f"gain{q}", None if out is None else (out * self.residual_mult).contiguous())

    def _source(self, ctx, x):
        """The tensor the streams are read from, and whether it is their common single row."""
        if ctx.streams_from is not None:
            return ctx.streams_from, True
        return x, False

    def _read(self, q: int, norm):
        if not isinstance(norm, RMSNorm):
            raise ValueError("residual streams are read through root-mean-square norms")
        return getattr(self, f"in{q}"), norm.weight, norm.eps

    def _write_back(self, ctx, x, y, q: int, read):
        """Sublayer ``q``'s result into the streams; returns the rows of the next read."""
        src, spread = self._source(ctx, x)
        last = read is None and self.streams > 1 and ctx.next_block is None
        out = torch.empty_like(y, dtype=ctx.rt.act_dtype) if read is not None else None
        total = torch.empty_like(y) if last else None
        ctx.ops.streams(src, self.streams, spread,
                        write=(y, getattr(self, f"scale{q}"), getattr(self, f"mix{q}"),
                               getattr(self, f"gain{q}")),
                        into=None if last else x, total=total, read=read, out=out)
        ctx.streams_from = None
        if last:
            ctx.streams_sum = total
        return out

    @staticmethod
    def _run(part, ctx, h, y):
        if getattr(part, "can_overwrite", False):
            part.forward(ctx, h, y, accumulate=False)
        else:
            part.forward(ctx, h, y.zero_())

    def forward(self, ctx, x, layer) -> None:
        n, dev = x.shape[0], x.device
        h, ctx.normed = ctx.normed, None
        if h is None:
            src, spread = self._source(ctx, x)
            h = torch.empty((n, self.width), device=dev, dtype=ctx.rt.act_dtype)
            ctx.ops.streams(src, self.streams, spread, read=self._read(1, layer.norm_mixer), out=h)
        y = torch.empty((n, self.width), device=dev, dtype=torch.float32)
        self._run(layer.mixer, ctx, h, y)
        nxt = ctx.next_block
        hand_over = nxt._read(1, ctx.next_norm) if isinstance(nxt, HyperConnectionsBlock) else None
        if layer.ffn is None:
            ctx.normed = self._write_back(ctx, x, y, 1, hand_over)
            return
        h = self._write_back(ctx, x, y, 1, self._read(2, layer.norm_ffn))
        y = torch.empty((n, self.width), device=dev, dtype=torch.float32)
        self._run(layer.ffn, ctx, h, y)
        ctx.normed = self._write_back(ctx, x, y, 2, hand_over)
