"""Causal attention whose keys and values are low-rank: only a latent per token is cached."""
from __future__ import annotations

import torch

from .base import MATRIX, VECTOR, KVRequest, Mixer, ParamSpec, register_part
from .linear import Linear
from .rotary import rotary_frequencies


@register_part("mixer", "latent_attention")
class LatentAttention(Mixer):
    """Multi-head attention over a shared latent.

    ``q = Wq h`` (``n_heads`` heads of ``head_dim``); ``c = rms(Wdown h) * latent_norm`` is the
    token's latent (``latent_dim`` numbers); head ``i`` has keys ``k_i = Wk_i c`` and values
    ``v_i = Wv_i c`` (``value_dim`` numbers); scores ``scale * q_i . k_i`` over positions ``j <=
    p``; with ``sink`` the softmax's denominator has one more term ``exp(sink_i)`` per head that
    belongs to no key; with ``gate`` head ``i``'s result is multiplied by ``sigmoid(Wgate h)_i``
    (``gate="each"``: every number of the concatenated heads by a logit of its own); ``Wout`` maps
    the concatenated heads back into the stream.

    ``q_latent_dim`` > 0: the queries go through a latent of their own, ``q = Wq_up (rms(Wq_down h)
    * q_norm)``.  ``rot_dim`` > 0: every query head has ``rot_dim`` more numbers, and ``Wdown h``
    as many more behind the latent (not normed), one key part shared by all heads; of both the
    first ``rot_dims`` are turned by position (pairs ``i, i + rot_dims/2``, ``parts/rotary.py`` with
    its frequency scaling), and their product joins the score in front of the scale.

    How it runs: one product gives ``[q or Wq_down h | Wdown h | gate logits]`` in fp32 (plus
    whatever else reads the same rows: ``extra_outputs`` columns that a feed-forward beside it
    picks up, e.g. its router's logits).  Keys and values are never formed: ``Wk_i`` moves to the
    query (``a_i = Wk_i^T q_i``, then ``a_i . c_j = q_i . k_i(j)``) and ``Wv_i`` behind the weighted
    sum (``Wv_i sum_j p_j c_j``), so every head attends over the same cached rows, which are key
    and value at once.  With rotated parts a cached row is ``[c | rotated key part]`` (the values
    are its first ``latent_dim`` numbers) and a query ``[a_i | rotated query part]``.  Norms, angles,
    scores, the softmax and the sink are fp32.
    """
    graph_safe = True
    can_overwrite = True

    def __init__(self, width: int, n_heads: int, head_dim: int, value_dim: int, latent_dim: int,
                 scale: float, eps: float, sink: bool = True, gate: bool | str = True, window: int = 0,
                 extra_outputs: int = 0, q_latent_dim: int = 0, rot_dim: int = 0,
                 rot_dims: int | None = None, rot_base: float = 10000.0,
                 rot_scaling: dict | None = None):
        self.width, self.n_heads = int(width), int(n_heads)
        self.head_dim, self.value_dim, self.latent_dim = int(head_dim), int(value_dim), int(latent_dim)
        self.scale, self.eps, self.window = float(scale), float(eps), int(window)
        self.has_sink, self.has_gate, self.gate_each = bool(sink), bool(gate), gate == "each"
        self.extra_outputs = int(extra_outputs)
        self.q_latent_dim, self.rot_dim = int(q_latent_dim or 0), int(rot_dim or 0)
        self.rot_dims = self.rot_dim if rot_dims is None else int(rot_dims)
        if self.rot_dims > self.rot_dim:
            raise ValueError("more turned dimensions than the rotated part has")
        self.rot_freq_host, self.rot_amplitude = rotary_frequencies(self.rot_dims, rot_base, rot_scaling) \
            if self.rot_dim else (None, 1.0)
        self.rot_freq = None
        self.row_dim = self.latent_dim + self.rot_dim          # a cached row, a query in its space
        # queries: all heads' plain parts, then all heads' rotated parts
        self.q_width = self.n_heads * self.head_dim
        q_outputs = self.n_heads * (self.head_dim + self.rot_dim)
        # columns of the fused projection's result
        self.col_latent = self.q_latent_dim or q_outputs
        self.col_gate = self.col_latent + self.row_dim
        n_gates = 0 if not self.has_gate else self.n_heads * (self.value_dim if self.gate_each else 1)
        self.col_extra = self.col_gate + n_gates
        # rows of zeros fill the projection up to a multiple of 8 outputs, so that its fp32 rows
        # start on 32-byte boundaries whatever the numbers of heads and extra outputs are
        self.proj_outputs = -(-(self.col_extra + self.extra_outputs) // 8) * 8
        self.proj = Linear(self.width, self.proj_outputs, bias=False)
        self.q_up = Linear(self.q_latent_dim, -(-q_outputs // 8) * 8, bias=False) \
            if self.q_latent_dim else None
        self.out = Linear(self.n_heads * self.value_dim, self.width, bias=False)
        self.latent_norm = self.key_up = self.value_up = self.sink = self.q_norm = None

    def children(self):
        own = {"proj": self.proj, "out": self.out}
        if self.q_up is not None:
            own["q_up"] = self.q_up
        return own

    def param_specs(self):
        specs = {
            "latent_norm": ParamSpec((self.latent_dim,), VECTOR),
            # per head, held for the products that run: [latent_dim, head_dim] = Wk_i transposed
            "key_up": ParamSpec((self.n_heads, self.latent_dim, self.head_dim), MATRIX),
            "value_up": ParamSpec((self.n_heads, self.value_dim, self.latent_dim), MATRIX),
        }
        if self.has_sink:
            specs["sink"] = ParamSpec((self.n_heads,), VECTOR)
        if self.q_latent_dim:
            specs["q_norm"] = ParamSpec((self.q_latent_dim,), VECTOR)
        return specs

    def bind(self, params, runtime) -> None:
        super().bind(params, runtime)
        if self.rot_freq_host is not None:
            self.rot_freq = self.rot_freq_host.to(runtime.device)

    def cache_request(self):
        return KVRequest(1, self.row_dim, self.window, planes=1)

    def forward(self, ctx, h: torch.Tensor, residual: torch.Tensor, accumulate: bool = True) -> None:
        lay, kv, ops = ctx.layout, ctx.kv, ctx.ops
        n, dev, act = lay.n_rows, h.device, ctx.rt.act_dtype
        fused = self.proj(ctx, h, out_dtype=torch.float32)
        ctx.shared_projection = (fused, self.col_extra)       # for a reader of the extra columns
        q = fused
        if self.q_up is not None:
            cq = torch.empty((n, self.q_latent_dim), device=dev, dtype=act)
            ops.rmsnorm(fused, self.q_norm, self.eps, cq)
            q = self.q_up(ctx, cq, out_dtype=torch.float32)
        a = torch.empty((n, self.n_heads * self.row_dim), device=dev, dtype=act)
        if self.rot_dim:
            ops.latent_rope_append(fused, self.col_latent, self.latent_norm, self.eps, self.rot_freq,
                                   self.rot_dim, self.rot_dims, self.rot_amplitude, q, self.q_width,
                                   a, self.n_heads, lay, kv, ctx.writes_cache)
        elif ctx.writes_cache:
            ops.latent_append(fused, self.col_latent, self.latent_norm, self.eps, lay, kv)
        ops.head_linear(q, 0, self.key_up, a, lay, out_stride=self.row_dim)
        mix = torch.empty((n, self.n_heads * self.latent_dim), device=dev, dtype=act)
        ops.attention_latent(a, lay, kv, self.n_heads, self.sink, mix, self.scale, self.window,
                             self.latent_dim)
        heads = torch.empty((n, self.n_heads * self.value_dim), device=dev, dtype=act)
        ops.head_linear(mix, 0, self.value_up, heads, lay, gate=fused if self.has_gate else None,
                        gate_col=self.col_gate, gate_each=self.gate_each)
        if accumulate:
            self.out(ctx, heads, residual=residual)
        else:
            self.out(ctx, heads, out=residual)
