"""Attention whose keys and values are rebuilt from a small latent vector per token, which is all
the cache keeps.

q = W_q x, per head [``head_dim`` plain | ``rot_dim`` rotated] elements.  W_dkv x has ``kv_rank`` +
``rot_dim`` rows: the first kv_rank, RMS-normed with a weight, are the latent c; the last rot_dim,
rotated by the token's position, are a key part k_r that all heads share.  Head h's key is
[W_uk,h c | k_r] and its value W_uv,h c, so

    score_h(i, j) = (q_plain,h(i) . W_uk,h c(j) + q_rot,h(i) . k_r(j)) * scale
                  = ([W_uk,h^T q_plain,h(i) | q_rot,h(i)] . [c(j) | k_r(j)]) * scale,
    out_h(i)      = W_uv,h sum_j p_h(i, j) c(j).

The second forms are what runs: the query is taken through the key map once, attention runs over
the cached rows [c | k_r] as ONE key head of kv_rank + rot_dim elements whose first kv_rank
elements double as the value, and the weighted latent goes through the value map.  A token costs
kv_rank + rot_dim cache elements whatever the number of heads.  Softmax over the keys the mask
shows ("causal", "window", "chunk" as in ``masked_attention``); norms, angles, scores and the softmax
are float32.  ``rotary_layout``: "halves" (element i of a rotated part turns with i + rot_dim / 2) or
"pairs" (2i with 2i + 1); the position encoding's ``amplitude`` multiplies cosine and sine.

``rot_dim`` 0 (no position encoding): there is no rotated part, the cache row is the latent alone.
``q_rank``: the queries go through a latent of their own, q = W_uq c_q with c_q = RMS norm of W_dq x with a
weight.  ``gate``: the heads' values side by side are multiplied element by element with sigmoid(W_g x)
before the output projection.

``own_latent`` off: the layer has no W_dkv and reads the rows that another layer of the same
kv_rank, rot_dim and rotation left in the cache its schedule entry names.
"""

from __future__ import annotations

from typing import Optional

import torch

from ..kernels import ops
from .base import Mixer
from .registry import POSITION_ENCODINGS, register_mixer
from .spec import PagedKVSpec, PartSpec, TensorSpec


@register_mixer("latent_attention")
class LatentAttention(Mixer):
    def __init__(self, ctx, prefix: str, hidden_size: int, num_heads: int, head_dim: int, rot_dim: int,
                 v_head_dim: int, kv_rank: int, scale: float, position_encoding: Optional[PartSpec], norm_eps: float,
                 mask: str = "causal", mask_size: Optional[int] = None, names: Optional[dict] = None,
                 rotary_layout: str = "halves", own_latent: bool = True, q_rank: Optional[int] = None,
                 gate: bool = False):
        if mask not in ("causal", "window", "chunk"):
            raise ValueError(f"mask {mask!r} is not known ('causal', 'window', 'chunk')")
        if mask != "causal" and (mask_size is None or int(mask_size) < 1):
            raise ValueError(f"a {mask} mask needs a positive mask_size")
        if rotary_layout not in ("halves", "pairs"):
            raise ValueError(f"rotary_layout {rotary_layout!r} is not known ('halves', 'pairs')")
        self.prefix = prefix
        self.rotary_layout, self.own_latent = rotary_layout, bool(own_latent)
        self.hidden_size, self.num_heads = int(hidden_size), int(num_heads)
        self.head_dim, self.rot_dim, self.v_head_dim = int(head_dim), int(rot_dim), int(v_head_dim)
        self.kv_rank, self.scale, self.norm_eps = int(kv_rank), float(scale), float(norm_eps)
        self.mask, self.mask_size = mask, None if mask == "causal" else int(mask_size)
        self.q_rank, self.gate = None if q_rank is None else int(q_rank), bool(gate)
        if not self.own_latent and (self.q_rank is not None or self.rot_dim == 0):
            raise ValueError("latent_attention: a layer that reads another's rows has plain queries and a rotated part")
        self.names = dict(q="q", down="dkv", latent_norm="dkv.norm", key_map="uk", value_map="uv", o="o", q_down="dq",
                          q_norm="dq.norm", q_up="uq", gate="g")
        self.names.update(names or {})
        self.position_encoding = None if position_encoding is None or not self.rot_dim \
            else POSITION_ENCODINGS.build(position_encoding, ctx)
        if getattr(self.position_encoding, "rotary_dim", 0) != self.rot_dim:
            raise ValueError(f"latent_attention: the rotation covers {getattr(self.position_encoding, 'rotary_dim', 0)} "
                             f"elements, the rotated part has {self.rot_dim}")
        self.amplitude = getattr(self.position_encoding, "amplitude", 1.0)
        self.out_dtype = ctx.dtype
        self.w_in = self.w_key = self.w_value = self.w_o = self.latent_norm = self.freq = None
        self.w_q_up = self.q_norm = None

    def tensor_specs(self):
        p, n, w = self.prefix, self.names, self.hidden_size
        h, d, r, e, c = self.num_heads, self.head_dim, self.rot_dim, self.v_head_dim, self.kv_rank
        if self.q_rank is None:
            specs = [TensorSpec(p + n["q"], (h * (d + r), w))]
        else:
            specs = [TensorSpec(p + n["q_down"], (self.q_rank, w)),
                     TensorSpec(p + n["q_norm"], (self.q_rank,), role="vector", init="one_plus_normal"),
                     TensorSpec(p + n["q_up"], (h * (d + r), self.q_rank))]
        if self.gate:
            specs.append(TensorSpec(p + n["gate"], (h * e, w)))
        if self.own_latent:
            specs += [TensorSpec(p + n["down"], (c + r, w)),
                      TensorSpec(p + n["latent_norm"], (c,), role="vector", init="one_plus_normal")]
        return specs + [TensorSpec(p + n["key_map"], (h * d, c)), TensorSpec(p + n["value_map"], (h * e, c)),
                        TensorSpec(p + n["o"], (w, h * e))]

    def load(self, tensors):
        p, n = self.prefix, self.names
        h, d, e, c = self.num_heads, self.head_dim, self.v_head_dim, self.kv_rank
        # one product gives [queries, or their latent | latent, rotated key part | gate]
        rows = [tensors[p + n["q" if self.q_rank is None else "q_down"]]]
        if self.own_latent:
            rows.append(tensors[p + n["down"]])
            self.latent_norm = tensors[p + n["latent_norm"]]
        if self.gate:
            rows.append(tensors[p + n["gate"]])
        self.w_in = torch.cat(rows, dim=0).contiguous() if len(rows) > 1 else rows[0]
        if self.q_rank is not None:
            self.q_norm, self.w_q_up = tensors[p + n["q_norm"]], tensors[p + n["q_up"]]
        # per head [K, N]: the key map takes a query's plain part [d] to the latent's size [c]; the
        # value map takes a weighted latent [c] to the head's value [e]
        self.w_key = tensors[p + n["key_map"]].view(h, d, c).contiguous()
        self.w_value = tensors[p + n["value_map"]].view(h, e, c).transpose(1, 2).contiguous()
        self.w_o = tensors[p + n["o"]]
        if self.rot_dim:
            self.freq = self.position_encoding.frequencies()

    def cache_spec(self):
        return PagedKVSpec(1, self.kv_rank + self.rot_dim, self.mask_size, v_head_dim=0,
                           mask="chunk" if self.mask == "chunk" else "window")

    def forward(self, x, step, cache):
        h, d, r, e, c = self.num_heads, self.head_dim, self.rot_dim, self.v_head_dim, self.kv_rank
        proj = ops.linear(x, self.w_in)
        t, width = proj.shape
        stored = cache.kv if cache.writes and self.own_latent else None
        rotation = dict(rotary_layout=self.rotary_layout, amplitude=self.amplitude)
        nq = h * (d + r)
        gate_col = (nq if self.q_rank is None else self.q_rank) + (c + r if self.own_latent else 0)
        if self.q_rank is not None:
            # the two latents, then the queries out of theirs
            c_q = ops.latent_rows(proj, 0, self.q_rank, self.q_norm, self.q_rank, c, r, self.latent_norm, self.norm_eps,
                                  self.freq, step.positions, stored, cache.slot_mapping, cache.page_size, self.out_dtype,
                                  **rotation)
            heads = ops.as_tensor(ops.linear(c_q, self.w_q_up))
            q = torch.empty(t, h, c, dtype=heads.dtype, device=heads.device) if r == 0 else \
                ops.latent_prepare(heads, h, d, r, c, None, self.norm_eps, self.freq, step.positions, None,
                                   cache.slot_mapping, cache.page_size, self.out_dtype, **rotation)
        else:
            heads = proj = ops.as_tensor(proj)
            q = ops.latent_prepare(proj, h, d, r, c, self.latent_norm, self.norm_eps, self.freq, step.positions, stored,
                                   cache.slot_mapping, cache.page_size, self.out_dtype, **rotation)
        row = heads.shape[1]
        ops.heads_linear(heads.as_strided((t, h, d), (row, d + r, 1)), self.w_key, q[:, :, :c])
        latent = ops.masked_attention(q, cache.kv, cache.attention_meta, self.scale, 1, c, cache.page_size,
                                      self.mask, self.mask_size, values_in_keys=True)
        o = torch.empty(t, h, e, dtype=heads.dtype, device=heads.device)
        ops.heads_linear(latent, self.w_value, o)
        o = o.view(t, h * e)
        if self.gate:
            ops.sigmoid_gate_(o, proj, gate_col)
        return ops.linear(o, self.w_o)
