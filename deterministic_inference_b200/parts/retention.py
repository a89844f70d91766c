"""Retention: a matrix state per head that shrinks by one constant a token, read without a softmax.

q = W_q x and k = W_k x (heads x ``head_dim``), v = W_v x and g = W_g x (heads x ``v_head_dim``), no
biases, one product of the concatenated weights.  The position encoding rotates the first
``rotary_dim`` elements of every q and k head in halves (element i with i + rotary_dim / 2); k is
multiplied by ``head_dim``^(-1/2) behind it.  Per head, with a state S [head_dim, v_head_dim] from zero:
    S <- decay_h S + k v^T;     o = S^T q.
A head's output is o / sqrt(mean(o^2) + ``norm_eps``), without a weight; the heads side by side, times
silu(g), go through W_o.  The state is float32 and lives in the
request's state slot; the rotation, the decays, the recurrence and the norm are float32 whatever
the engine's storage type.
"""

from __future__ import annotations

from typing import Optional

import torch

from ..kernels import ops
from .base import Mixer
from .registry import POSITION_ENCODINGS, register_mixer
from .spec import PartSpec, StateSpec, TensorSpec


@register_mixer("retention")
class Retention(Mixer):
    # the kernels take the sequences' state slots from the step's device metadata, and a
    # sequence on state slot 0 (padding) starts from zero and stores nothing
    state_on_device = True

    def __init__(self, ctx, prefix: str, hidden_size: int, num_heads: int, head_dim: int, v_head_dim: int,
                 decay, norm_eps: float, position_encoding: Optional[PartSpec] = None,
                 names: Optional[dict] = None):
        self.prefix = prefix
        self.hidden_size, self.num_heads = int(hidden_size), int(num_heads)
        self.head_dim, self.v_head_dim = int(head_dim), int(v_head_dim)
        self.norm_eps = float(norm_eps)
        self.decay_list = [float(d) for d in decay]
        if len(self.decay_list) != self.num_heads or not all(0.0 <= d <= 1.0 for d in self.decay_list):
            raise ValueError(f"retention: {self.num_heads} heads need as many decays in [0, 1], got {list(decay)!r}")
        self.names = dict(q="q", k="k", v="v", g="g", o="o")
        self.names.update(names or {})
        self.position_encoding = None if position_encoding is None \
            else POSITION_ENCODINGS.build(position_encoding, ctx)
        self.rotary_dim = getattr(self.position_encoding, "rotary_dim", 0)
        if self.rotary_dim > self.head_dim or getattr(self.position_encoding, "amplitude", 1.0) != 1.0:
            raise ValueError("retention: the rotation covers more than a head, or scales it")
        self.device, self.out_dtype = ctx.device, ctx.dtype
        self.w_in = self.w_o = self.freq = self.decay = None

    def tensor_specs(self):
        p, n, w = self.prefix, self.names, self.hidden_size
        qk, v = self.num_heads * self.head_dim, self.num_heads * self.v_head_dim
        return [TensorSpec(p + n["q"], (qk, w)), TensorSpec(p + n["k"], (qk, w)), TensorSpec(p + n["v"], (v, w)),
                TensorSpec(p + n["g"], (v, w)), TensorSpec(p + n["o"], (w, v))]

    def load(self, tensors):
        p, n = self.prefix, self.names
        self.w_in = torch.cat([tensors[p + n[x]] for x in ("q", "k", "v", "g")], dim=0).contiguous()
        self.w_o = tensors[p + n["o"]]
        self.decay = torch.tensor(self.decay_list, dtype=torch.float32).to(self.device)
        if self.rotary_dim:
            self.freq = self.position_encoding.frequencies()

    def cache_spec(self):
        # one row of a slot: the heads' states [H, D, E]
        return StateSpec((self.num_heads * self.head_dim * self.v_head_dim,), "float32")

    def forward(self, x, step, cache):
        y = ops.retention(ops.linear(x, self.w_in), self.decay, self.freq, cache.state, step, self.num_heads,
                          self.head_dim, self.v_head_dim, self.norm_eps, self.out_dtype)
        return ops.linear(y, self.w_o)
