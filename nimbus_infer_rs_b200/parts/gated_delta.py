"""A linear-recurrent mixer: the gated delta rule with a decay per key channel."""
from __future__ import annotations

import torch

from .base import MATRIX, VECTOR, Mixer, ParamSpec, StateRequest, register_part
from .linear import Linear


@register_part("mixer", "gated_delta_rule")
class GatedDeltaRule(Mixer):
    """Per head a state matrix ``S`` (``head_dim`` key channels x ``value_dim`` value channels, fp32,
    zero at the start of a sequence) that every token decays, corrects and then reads:

        S <- diag(g) S,    u = beta (v - S^T k),    S <- S + k u^T,    o = S^T q

    ``q, k`` (``n_kv_heads`` heads; head ``h`` uses head ``h // (n_heads / n_kv_heads)``) and ``v``
    (``n_heads`` heads) are projections that each pass a short causal convolution over time per
    channel (``taps`` numbers a channel, the last one meets the current token, no bias) and a
    silu; ``q`` and ``k`` are then brought to unit length per head (``x / sqrt(sum x^2 + key_eps)``)
    and ``q`` is multiplied by ``head_dim^(-1/2)``.  ``beta = sigmoid(Wb h)``, one per head; ``g =
    exp(-exp(A_h) softplus(Wa2 (Wa1 h) + dt_bias))``, one per head and key channel.  Each head's
    ``o`` is divided by its root mean square (``eps`` inside the root), multiplied by the weight
    ``norm`` (``value_dim`` numbers, shared by the heads) and by ``sigmoid(Wg2 (Wg1 h))``; ``Wout``
    maps the heads side by side back.

    How it runs: one product gives ``[q | k | v | beta logits | Wa1 h | Wg1 h]`` in fp32; one small
    product maps the two low-rank columns up; the recurrence's kernels do everything else in fp32,
    the convolution included, and leave the matrices and the convolution's last ``taps - 1`` inputs
    in the sequence's state row.  Nothing grows with the sequence.
    """
    graph_safe = True
    can_overwrite = True

    def __init__(self, width: int, n_heads: int, n_kv_heads: int, head_dim: int, value_dim: int,
                 taps: int, decay_rank: int, gate_rank: int, eps: float, key_eps: float = 1e-6):
        self.width, self.n_heads, self.n_kv_heads = int(width), int(n_heads), int(n_kv_heads)
        self.head_dim, self.value_dim, self.taps = int(head_dim), int(value_dim), int(taps)
        self.eps, self.key_eps = float(eps), float(key_eps)
        if self.n_heads % self.n_kv_heads:
            raise ValueError("n_heads must be divisible by n_kv_heads")
        if self.taps < 1:
            raise ValueError(f"a convolution of {self.taps} taps")
        self.qk_width = self.n_kv_heads * self.head_dim
        self.v_width = self.n_heads * self.value_dim
        self.channels = 2 * self.qk_width + self.v_width            # of the convolution
        # the two low-rank maps run as one product of two "heads" of one size
        self.rank = max(int(decay_rank), int(gate_rank))
        self.up_width = max(self.n_heads * self.head_dim, self.v_width)
        # columns of the fused projection's result; the low-rank ones on a multiple of 8
        self.col_beta = self.channels
        self.col_low = -(-(self.col_beta + self.n_heads) // 8) * 8
        self.proj = Linear(self.width, -(-(self.col_low + 2 * self.rank) // 8) * 8, bias=False)
        self.out = Linear(self.v_width, self.width, bias=False)
        self.conv = self.up = self.a_log = self.dt_bias = self.norm = None

    def children(self):
        return {"proj": self.proj, "out": self.out}

    def param_specs(self):
        return {"conv": ParamSpec((self.channels, self.taps), VECTOR),
                "up": ParamSpec((2, self.up_width, self.rank), MATRIX),
                "a_log": ParamSpec((self.n_heads,), VECTOR),
                "dt_bias": ParamSpec((self.n_heads * self.head_dim,), VECTOR),
                "norm": ParamSpec((self.value_dim,), VECTOR)}

    @property
    def matrix_elements(self) -> int:
        return self.n_heads * self.head_dim * self.value_dim

    def state_request(self):
        # the matrices, then the convolution's inputs
        n = self.matrix_elements + (self.taps - 1) * self.channels
        return StateRequest(-(-n // 4) * 4)

    def forward(self, ctx, h: torch.Tensor, residual: torch.Tensor, accumulate: bool = True) -> None:
        lay, ops = ctx.layout, ctx.ops
        n, dev, act = lay.n_rows, h.device, ctx.rt.act_dtype
        m = self.matrix_elements
        matrices = ctx.state[:, :m]
        inputs = ctx.state[:, m:m + (self.taps - 1) * self.channels]
        fused = self.proj(ctx, h, out_dtype=torch.float32)
        low = torch.empty((n, 2 * self.up_width), device=dev, dtype=torch.float32)
        ops.head_linear(fused, self.col_low, self.up, low, lay)
        o = torch.empty((n, self.v_width), device=dev, dtype=act)
        ops.gated_delta(fused, 0, self.conv, self.taps, inputs, fused, self.col_beta, low, 0,
                        self.up_width, self.a_log, self.dt_bias, self.norm, self.eps, self.key_eps,
                        lay, matrices, self.n_heads, self.n_kv_heads, self.head_dim, self.value_dim, o)
        if accumulate:
            self.out(ctx, o, residual=residual)
        else:
            self.out(ctx, o, out=residual)
