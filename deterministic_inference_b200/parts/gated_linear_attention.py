"""Gated linear attention: a matrix state per head whose rows decay by a number of their own every token.

q = W_q x and k = W_k x (heads x ``head_dim``), v = W_v x and g = W_g x (heads x ``v_head_dim``), no
biases; q is multiplied by ``head_dim``^(-1/2).  A decay per key channel: alpha = sigmoid(z)^(1 / ``tau``)
with z = W_a2 (W_a1 x) + b, a map of rank ``decay_rank``.  Per head, with a state S [head_dim, v_head_dim]
from zero:
    S <- diag(alpha) S + k v^T;     o = S^T q.
A head's output is o / sqrt(mean(o^2) + ``norm_eps``) times a weight of size v_head_dim that the heads
share; the heads side by side, times silu(g), go through W_o.  The state is float32 and lives in the
request's state slot; the decay map's products, the decays, the recurrence and the norm are float32
whatever the engine's storage type.
"""

from __future__ import annotations

from typing import Optional

import torch

from ..kernels import gemm_bf16, ops
from .base import Mixer
from .registry import register_mixer
from .spec import StateSpec, TensorSpec


@register_mixer("gated_linear_attention")
class GatedLinearAttention(Mixer):
    # the kernels take the sequences' state slots from the step's device metadata, and a
    # sequence on state slot 0 (padding) starts from zero and stores nothing
    state_on_device = True

    def __init__(self, ctx, prefix: str, hidden_size: int, num_heads: int, head_dim: int, v_head_dim: int,
                 decay_rank: int, tau: float, norm_eps: float, names: Optional[dict] = None):
        if not float(tau) > 0:
            raise ValueError(f"gated_linear_attention: tau {tau!r} must be positive")
        self.prefix = prefix
        self.hidden_size, self.num_heads = int(hidden_size), int(num_heads)
        self.head_dim, self.v_head_dim = int(head_dim), int(v_head_dim)
        self.decay_rank, self.tau, self.norm_eps = int(decay_rank), float(tau), float(norm_eps)
        self.names = dict(q="q", k="k", v="v", g="g", o="o", a1="a1", a2="a2", a2_bias="a2.b", norm="norm")
        self.names.update(names or {})
        self.out_dtype = ctx.dtype
        self.w_in = self.w_o = self.a2_t = self.a2_bias = self.norm_weight = None

    def tensor_specs(self):
        p, n, w = self.prefix, self.names, self.hidden_size
        qk, v = self.num_heads * self.head_dim, self.num_heads * self.v_head_dim
        return [TensorSpec(p + n["q"], (qk, w)), TensorSpec(p + n["k"], (qk, w)), TensorSpec(p + n["v"], (v, w)),
                TensorSpec(p + n["g"], (v, w)), TensorSpec(p + n["a1"], (self.decay_rank, w)),
                TensorSpec(p + n["a2"], (qk, self.decay_rank)),
                TensorSpec(p + n["a2_bias"], (qk,), role="vector", init="normal"),
                TensorSpec(p + n["norm"], (self.v_head_dim,), role="vector", init="one_plus_normal"),
                TensorSpec(p + n["o"], (w, v))]

    @property
    def _proj_width(self) -> int:
        return 2 * self.num_heads * (self.head_dim + self.v_head_dim)

    def load(self, tensors):
        p, n = self.prefix, self.names
        rows = [tensors[p + n[x]] for x in ("q", "k", "v", "g", "a1")]
        have = sum(r.shape[0] for r in rows)
        if have % 8:                 # (filled up to a multiple of 8 with zeros)
            rows.append(torch.zeros(8 - have % 8, self.hidden_size, dtype=rows[0].dtype, device=rows[0].device))
        self.w_in = torch.cat(rows, dim=0).contiguous()
        self.w_o = tensors[p + n["o"]]
        self.a2_t, self.a2_bias = tensors[p + n["a2"]].t().contiguous(), tensors[p + n["a2_bias"]]
        self.norm_weight = tensors[p + n["norm"]]

    def cache_spec(self):
        # one row of a slot: the heads' states [H, D, E]
        return StateSpec((self.num_heads * self.head_dim * self.v_head_dim,), "float32")

    def forward(self, x, step, cache):
        width = self._proj_width
        if x.dtype == torch.bfloat16 and x.shape[0] > gemm_bf16.MAX_ROWS and width % 8 == 0:
            # many rows: q, k, v and g as stored bfloat16 rows, the decay map's input as float32 sums
            proj = ops.linear(x, self.w_in[:width])
            hidden, col = ops.linear(x, self.w_in[width:], out_dtype=torch.float32), 0
        else:
            # few rows: one product, whose float32 sums the kernels read (and round where a stored
            # projection would be rounded)
            proj = hidden = ops.linear(x, self.w_in, out_dtype=torch.float32 if x.dtype != torch.float32 else None)
            col = width
        y = ops.gated_linear_attention(proj, hidden, col, self.a2_t, self.a2_bias, self.tau, self.norm_weight,
                                       cache.state, step, self.num_heads, self.head_dim, self.v_head_dim,
                                       self.norm_eps, self.out_dtype)
        return ops.linear(y, self.w_o)
