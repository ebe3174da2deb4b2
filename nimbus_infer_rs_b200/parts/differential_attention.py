"""Grouped-query attention whose heads are the difference of two attention maps over one set of
values."""
from __future__ import annotations

import math

import torch

from .base import VECTOR, KVRequest, Mixer, ParamSpec, register_part
from .linear import Linear


@register_part("mixer", "differential_attention")
class DifferentialAttention(Mixer):
    """``n_heads`` query heads over ``n_kv_heads`` key/value heads (query head ``h`` uses key head
    ``h // (n_heads / n_kv_heads)``).  A query and a key head consist of two maps of ``head_dim``
    numbers each, side by side; a value head has ``value_dim`` numbers, shared by both maps.

    Map ``a`` is an attention of its own, scores ``scale * q_a . k_a``, softmax over what the
    position sees: every ``j <= i``, or with ``window`` > 0 those with ``i - j < window``.  With
    ``A_1, A_2`` the maps' results and one number per layer,

        ``lam = exp(sum lq1 * lk1) - exp(sum lq2 * lk2) + diff``,

    a head's result is ``u / sqrt(mean(u^2) + eps) * (1 - diff)``, ``u = A_1 - lam * A_2`` (no
    weight).  ``Wo`` maps the concatenated heads back.  No biases, no positions.

    One product gives ``[q | k | v]`` in fp32; keys and values go to the paged store (two planes of
    one store when ``value_dim = 2 head_dim``, else a store each; a window gives its pages back);
    both maps, their difference, its norm and the factor are one kernel.
    """
    graph_safe = True
    can_overwrite = True

    def __init__(self, width: int, n_heads: int, n_kv_heads: int, head_dim: int, scale: float,
                 diff: float, value_dim: int | None = None, window: int = 0, eps: float = 1e-6):
        self.width, self.n_heads, self.n_kv_heads = int(width), int(n_heads), int(n_kv_heads)
        self.head_dim = int(head_dim)
        self.value_dim = int(value_dim) if value_dim else 2 * self.head_dim
        if self.n_heads % self.n_kv_heads:
            raise ValueError("n_heads must be divisible by n_kv_heads")
        self.scale, self.diff = float(scale), float(diff)
        self.window, self.eps = int(window), float(eps)
        self.one_store = self.value_dim == 2 * self.head_dim
        self.q_width = self.n_heads * 2 * self.head_dim
        self.col_k = self.q_width
        self.col_v = self.col_k + self.n_kv_heads * 2 * self.head_dim
        outputs = self.col_v + self.n_kv_heads * self.value_dim
        # rows of zeros fill the fused projection up to a multiple of 8 outputs
        self.proj = Linear(self.width, -(-outputs // 8) * 8, bias=False)
        self.out = Linear(self.n_heads * self.value_dim, self.width, bias=False)
        self.lq1 = self.lk1 = self.lq2 = self.lk2 = None
        self.lam = None

    def children(self):
        return {"proj": self.proj, "out": self.out}

    def param_specs(self):
        return {n: ParamSpec((self.head_dim,), VECTOR) for n in ("lq1", "lk1", "lq2", "lk2")}

    def bind(self, params, runtime) -> None:
        super().bind(params, runtime)
        if self.lq1 is not None:
            # a constant of the layer: worked out once, on the host
            a, b, c, d = (t.detach().to("cpu", torch.float64) for t in
                          (self.lq1, self.lk1, self.lq2, self.lk2))
            self.lam = math.exp(float((a * b).sum())) - math.exp(float((c * d).sum())) + self.diff

    def cache_request(self):
        return KVRequest(self.n_kv_heads, 2 * self.head_dim, self.window,
                         planes=2 if self.one_store else 1)

    def extra_cache_requests(self):
        return () if self.one_store else (KVRequest(self.n_kv_heads, self.value_dim, self.window,
                                                    planes=1),)

    def forward(self, ctx, h: torch.Tensor, residual: torch.Tensor, accumulate: bool = True) -> None:
        lay, ops = ctx.layout, ctx.ops
        n, dev, act = lay.n_rows, h.device, ctx.rt.act_dtype
        keys = ctx.kv
        values = keys if self.one_store else ctx.kv_extra[0]
        fused = self.proj(ctx, h, out_dtype=torch.float32)
        q = torch.empty((n, self.q_width), device=dev, dtype=act)
        ops.qkv_norm_rope_append(fused, 0, self.col_k, self.col_v, None, None, 0.0, None, 0, 1.0, lay,
                                 keys, values, self.n_heads, self.value_dim, q, ctx.writes_cache)
        attn = torch.empty((n, self.n_heads * self.value_dim), device=dev, dtype=act)
        ops.attention_differential(q, lay, keys, values, self.n_heads, attn, self.scale, self.window,
                                   self.lam, 1.0 - self.diff, self.eps)
        if accumulate:
            self.out(ctx, attn, residual=residual)
        else:
            self.out(ctx, attn, out=residual)
