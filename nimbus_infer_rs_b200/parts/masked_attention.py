"""Grouped-query attention with biases, rotated (and optionally normed) queries and keys, capped
scores, a mask by window or by block, a sink and a gate per head: each of them optional."""
from __future__ import annotations

import torch

from .base import VECTOR, KVRequest, Mixer, ParamSpec, register_part
from .linear import Linear
from .rotary import rotary_frequencies


@register_part("mixer", "masked_attention")
class MaskedAttention(Mixer):
    """``n_heads`` query heads over ``n_kv_heads`` key/value heads (query head ``h`` uses key head
    ``h // (n_heads / n_kv_heads)``), keys of ``head_dim`` numbers and values of ``value_dim``.

    One product gives ``[q | k | v | gate logits]`` in fp32 (with ``bias``, a bias on each).  With
    ``qk_norm="head"`` (or ``True``) queries and keys get a per-head RMS norm (weights ``q_norm`` /
    ``k_norm`` of ``head_dim`` numbers, shared by the heads; ``eps`` inside the root), with
    ``qk_norm="whole"`` all heads' queries are normed together, and all heads' keys (weights of
    those sizes); then, with ``rot_dims`` > 0, the first ``rot_dims`` numbers of every query and
    key head are turned by position, dimension ``i`` paired with ``i + rot_dims / 2``
    (``parts/rotary.py``, with its frequency scaling ``rot_scaling``); values get neither.

    A score is ``scale * q . k`` and, with ``softcap`` > 0, then ``softcap * tanh(score /
    softcap)``.  What position ``i`` sees among ``j <= i``:

    * ``window`` > 0: ``i - j < window``, and besides those every ``j < keep_first`` (the
      sequence's first tokens stay visible at their true positions);
    * ``chunk`` > 0: only ``j`` with ``floor(j / chunk) == floor(i / chunk)``, blocks counted from
      the sequence's position 0 whatever the step's cut;
    * neither: every ``j <= i``.

    With ``sink`` the softmax's denominator has one more term ``exp(sink_h)`` per head (no key, no
    value, neither scaled nor capped); ``sink="zero"``: ``sink_h = 0``, not a parameter.  With
    ``gate`` head ``h``'s result is multiplied by ``sigmoid(Wg x)_h``, one logit per head from the
    mixer's own input.  ``Wo`` (with ``out_bias``, and a bias) maps the concatenated heads back.

    ``own_keys=False``: the mixer projects queries only and reads the keys (as they are cached,
    normed and turned) and values of another layer's store (``LayerSpec.cache_from``).

    Storage: a paged store of two planes (keys and values, each with its own size).  A store
    with a window gives back the pages that no later token sees, except those of the kept first
    tokens; a block mask never looks further back than ``chunk`` tokens, so its pages are given
    back like a window's.
    """
    graph_safe = True
    can_overwrite = True

    def __init__(self, width: int, n_heads: int, n_kv_heads: int, head_dim: int, scale: float,
                 value_dim: int | None = None, eps: float = 1e-6, qk_norm: bool | str = False,
                 softcap: float = 0.0, window: int = 0, keep_first: int = 0, chunk: int = 0,
                 sink: bool | str = False, gate: bool = False, rot_dims: int = 0,
                 rot_base: float = 10000.0, rot_scaling: dict | None = None, bias: bool = False,
                 out_bias: bool = False, own_keys: bool = True):
        self.width, self.n_heads, self.n_kv_heads = int(width), int(n_heads), int(n_kv_heads)
        self.head_dim = int(head_dim)
        self.value_dim = int(value_dim) if value_dim else self.head_dim
        self.scale, self.eps, self.softcap = float(scale), float(eps), float(softcap or 0.0)
        self.window, self.keep_first, self.chunk = int(window), int(keep_first), int(chunk)
        if self.n_heads % self.n_kv_heads:
            raise ValueError("n_heads must be divisible by n_kv_heads")
        if self.window > 0 and self.chunk > 0:
            raise ValueError("a mask is a window or a block, not both")
        if self.window <= 0:
            self.keep_first = 0             # without a window every first token is seen anyway
        if qk_norm not in (False, None, True, "head", "whole") or sink not in (False, None, True, "zero"):
            raise ValueError(f"qk_norm={qk_norm!r}: head or whole; sink={sink!r}: True or zero")
        self.has_norm, self.norm_whole = bool(qk_norm), qk_norm == "whole"
        self.has_sink, self.sink_zero, self.has_gate = bool(sink), sink == "zero", bool(gate)
        self.own_keys = bool(own_keys)
        self.rot_dims = int(rot_dims)
        if self.rot_dims > self.head_dim:
            raise ValueError("more rotated dimensions than the head has")
        self.rot_freq_host, self.rot_amplitude = (None, 1.0) if not self.rot_dims else \
            rotary_frequencies(self.rot_dims, rot_base, rot_scaling)
        self.rot_freq = None
        self.q_width = self.n_heads * self.head_dim
        self.k_width = self.n_kv_heads * self.head_dim
        self.v_width = self.n_kv_heads * self.value_dim
        self.col_k = self.q_width
        self.col_v = self.col_k + (self.k_width if self.own_keys else 0)
        self.col_gate = self.col_v + (self.v_width if self.own_keys else 0)
        outputs = self.col_gate + (self.n_heads if self.has_gate else 0)
        # rows of zeros fill the fused projection up to a multiple of 8 outputs
        self.proj = Linear(self.width, -(-outputs // 8) * 8, bias="required" if bias else False)
        self.out = Linear(self.n_heads * self.value_dim, self.width,
                          bias="required" if out_bias else False)
        self.q_norm = self.k_norm = self.sink = None

    def children(self):
        return {"proj": self.proj, "out": self.out}

    def param_specs(self):
        specs = {}
        if self.has_norm:
            whole = self.norm_whole
            specs["q_norm"] = ParamSpec((self.q_width if whole else self.head_dim,), VECTOR)
            if self.own_keys:
                specs["k_norm"] = ParamSpec((self.k_width if whole else self.head_dim,), VECTOR)
        if self.has_sink and not self.sink_zero:
            specs["sink"] = ParamSpec((self.n_heads,), VECTOR)
        return specs

    def bind(self, params, runtime) -> None:
        super().bind(params, runtime)
        if self.rot_freq_host is not None:
            self.rot_freq = self.rot_freq_host.to(runtime.device)
        if self.sink_zero:
            self.sink = torch.zeros(self.n_heads, dtype=torch.float32, device=runtime.device)

    def _look_back(self) -> int:
        return self.window if self.window > 0 else self.chunk

    def cache_request(self):
        return KVRequest(self.n_kv_heads, self.head_dim, self._look_back(), keep_first=self.keep_first,
                         value_dim=None if self.value_dim == self.head_dim else self.value_dim)

    def forward(self, ctx, h: torch.Tensor, residual: torch.Tensor, accumulate: bool = True) -> None:
        lay, ops = ctx.layout, ctx.ops
        n, dev, act = lay.n_rows, h.device, ctx.rt.act_dtype
        kv = ctx.kv
        fused = self.proj(ctx, h, out_dtype=torch.float32)
        q = torch.empty((n, self.q_width), device=dev, dtype=act)
        ops.qkv_norm_rope_append(fused, 0, self.col_k, self.col_v, self.q_norm, self.k_norm,
                                 self.eps, self.rot_freq, self.rot_dims, self.rot_amplitude, lay,
                                 kv, kv, self.n_heads, self.value_dim, q,
                                 ctx.writes_cache and self.own_keys, self.norm_whole)
        attn = torch.empty((n, self.n_heads * self.value_dim), device=dev, dtype=act)
        ops.attention_masked(q, lay, kv, kv, self.n_heads, self.sink, attn, self.scale,
                             self.softcap, self.window, self.keep_first, self.chunk,
                             fused if self.has_gate else None, self.col_gate)
        if accumulate:
            self.out(ctx, attn, residual=residual)
        else:
            self.out(ctx, attn, out=residual)
