"""A plain, slow implementation of the Nedupel design: whole sequences, no cache, no batches,
float64 by default, one function per mechanism, written from the design's equations.  It shares
no code with the package; the tests compare the package with it.

Notation: n tokens, width W.  ``w`` maps tensor names to tensors, ``p`` is a part's prefix
("l3.mix." and the like), ``c`` the part's entry of config.json.  ``rnd`` rounds what a
bfloat16 engine stores (a yardstick for its tests); by default nothing is rounded.

The stream starts as embed[token] * s_e.  A layer is x <- x + m mixer(norm1(x)), then
x <- x + m ff(norm2(x)), m one constant of the model, norms with weights around zero.  Mixers:
"latent_attention" (keys and values from a small latent vector per token, a rotated key part
shared by the heads; a layer may use the latents of an earlier one) and "retention" (a matrix
state per head that shrinks by a constant every token).  The feed-forward is dense with a squared relu, or a
mixture of experts whose choice is a table of the token ids.
"""

from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import torch

DT = torch.float64


def read_model_dir(model_dir, dtype=DT):
    """(config dict, {name: tensor}) of a folder with config.json and model.safetensors."""
    model_dir = Path(model_dir)
    cfg = json.loads((model_dir / "config.json").read_text())
    raw = (model_dir / "model.safetensors").read_bytes()
    (n,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8:8 + n])
    data = raw[8 + n:]
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32}
    out = {}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        a, b = meta["data_offsets"]
        t = torch.frombuffer(bytearray(data[a:b]), dtype=kinds[meta["dtype"]]).reshape(meta["shape"])
        out[name] = t.to(dtype) if t.is_floating_point() else t
    return cfg, out


def _keep(x):
    return x


def as_stored_bf16(x):
    return x.to(torch.bfloat16).to(x.dtype)


# ---- small functions -------------------------------------------------------------------------

def unit_rms(x, eps):
    """x over its root mean square over the last dimension, eps inside the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def around_zero_norm(x, weight, eps):
    return unit_rms(x, eps) * (1.0 + weight)


def silu(z):
    return z * torch.sigmoid(z)


# ---- rotations ---------------------------------------------------------------------------------

def plain_frequencies(dims, base):
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def yarn_frequencies(dims, base, scaling):
    """(frequencies, factor on cos and sin).  A pair that turns more than ``fast`` times over
    ``original`` positions keeps its frequency, one that turns less than ``slow`` times has it divided
    by ``factor``, and between the two the pair's index decides linearly."""
    if scaling is None:
        return plain_frequencies(dims, base), 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def index_of(turns):       # the (fractional) pair index whose frequency turns so often
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(float(scaling["fast"]))), 0)
    hi = min(math.ceil(index_of(float(scaling["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(plain_frequencies(dims, base)):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * r + f * (1.0 - r))
    return out, 0.1 * math.log(factor) + 1.0


def turn(u, v, positions, freqs, size=1.0):
    """(u cos a - v sin a, v cos a + u sin a) with a = position * f_i; u, v [n, heads, pairs]."""
    a = positions.to(u.dtype)[:, None] * torch.tensor(freqs, dtype=u.dtype)[None, :]
    cos, sin = size * torch.cos(a)[:, None, :], size * torch.sin(a)[:, None, :]
    return u * cos - v * sin, v * cos + u * sin


def rotate_pairs(x, positions, freqs, size):
    """x [n, heads, 2 pairs]: element 2i turns with element 2i + 1."""
    u, v = turn(x[..., 0::2], x[..., 1::2], positions, freqs, size)
    return torch.stack([u, v], dim=-1).flatten(-2)


def rotate_halves(x, positions, freqs):
    """x [n, heads, D]: element i turns with element i + pairs; elements from 2 pairs on pass."""
    half = len(freqs)
    u, v = turn(x[..., :half], x[..., half:2 * half], positions, freqs)
    return torch.cat([u, v, x[..., 2 * half:]], dim=-1)


# ---- mixer "latent_attention" ---------------------------------------------------------------------

def latent_rows(h, w, p, c, eps, rnd=_keep):
    """(latents [n, rank], rotated key part [n, rot_dim]) of every token: all that a cache keeps."""
    rank = c["kv_rank"]
    down = rnd(h @ w[p + "dkv"].T)
    latent = unit_rms(down[:, :rank], eps) * w[p + "dkv.norm"]
    freqs, size = yarn_frequencies(c["rot"]["dims"], float(c["rot"]["base"]), c["rot"].get("scaling"))
    key = rotate_pairs(down[:, None, rank:], torch.arange(h.shape[0]), freqs, size)[:, 0]
    return rnd(latent), rnd(key)


def latent_attention(h, w, p, c, rows, rnd=_keep):
    """``rows``: the latents and rotated key parts the layer reads (its own or another layer's)."""
    n, heads, d, r, e = h.shape[0], c["heads"], c["dim"], c["rot_dim"], c["vdim"]
    latent, key_rot = rows
    q = rnd(h @ w[p + "q"].T).reshape(n, heads, d + r)
    freqs, size = yarn_frequencies(c["rot"]["dims"], float(c["rot"]["base"]), c["rot"].get("scaling"))
    q_rot = rnd(rotate_pairs(q[..., d:], torch.arange(n), freqs, size))
    k = rnd(latent @ w[p + "uk"].T).reshape(n, heads, d)
    v = rnd(latent @ w[p + "uv"].T).reshape(n, heads, e)
    future = torch.ones(n, n, dtype=torch.bool).triu(1)
    out = torch.zeros(n, heads, e, dtype=h.dtype)
    for i in range(heads):
        s = (q[:, i, :d] @ k[:, i].T + q_rot[:, i] @ key_rot.T) * float(c["scale"])
        out[:, i] = torch.softmax(s.masked_fill(future, -math.inf), dim=-1) @ v[:, i]
    return rnd(rnd(out).reshape(n, heads * e) @ w[p + "o"].T)


# ---- mixer "retention" ------------------------------------------------------------------------------

def retention_recurrence(q, k, v, decay):
    """q, k [n, H, D], v [n, H, E], decay [H].  Per head from S = 0 [D, E]: S <- decay S + k v^T; o = S^T q."""
    n, heads, d = q.shape
    out = torch.zeros(n, heads, v.shape[-1], dtype=q.dtype)
    for i in range(heads):
        s = torch.zeros(d, v.shape[-1], dtype=q.dtype)
        for t in range(n):
            s = float(decay[i]) * s + torch.outer(k[t, i], v[t, i])
            out[t, i] = s.T @ q[t, i]
    return out


def retention(h, w, p, c, eps, rnd=_keep):
    n, heads, d, e = h.shape[0], c["heads"], c["dim"], c["vdim"]
    pos = torch.arange(n)
    freqs = plain_frequencies(c["rot"]["dims"], float(c["rot"]["base"]))
    q = rotate_halves(rnd(h @ w[p + "q"].T).reshape(n, heads, d), pos, freqs)
    k = rotate_halves(rnd(h @ w[p + "k"].T).reshape(n, heads, d), pos, freqs) * d ** -0.5
    v = rnd(h @ w[p + "v"].T).reshape(n, heads, e)
    o = unit_rms(retention_recurrence(q, k, v, c["decay"]), eps).reshape(n, heads * e)
    return rnd(rnd(o * silu(rnd(h @ w[p + "g"].T))) @ w[p + "o"].T)


# ---- feed-forward ---------------------------------------------------------------------------------

def squared_relu_feed_forward(h, w, p, rnd=_keep):
    z = torch.relu(rnd(h @ w[p + "up"].T))
    return rnd(rnd(z * z) @ w[p + "down"].T)


def expert(h, w, p, limit, rnd=_keep):
    g = torch.clamp(rnd(h @ w[p + "gate"].T), max=limit)
    u = torch.clamp(rnd(h @ w[p + "up"].T), -limit, limit)
    return rnd(rnd(g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T)


def table_experts(h, w, p, c, tokens, rnd=_keep):
    table, top = w[p + "table"], c["router"]["top"]
    out = torch.zeros_like(h)
    for t, token in enumerate(tokens):
        for j in range(top):
            e = int(table[int(token), j])
            out[t] = out[t] + expert(h[t:t + 1], w, f"{p}e{e}.", float(c["expert"]["limit"]), rnd)[0] / top
    return out


# ---- the model ------------------------------------------------------------------------------------

def forward(cfg, w, tokens, rnd=_keep, layers_out=None):
    """Logits [n, vocab] of one sequence.  ``layers_out``: a list that receives the residual stream
    after every layer."""
    eps, m = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    tokens = [int(t) for t in tokens]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * float(cfg["embedding"]["scale"])
    rows = {}
    for i, layer in enumerate(cfg["layers"]):
        p, c = f"l{i}.", layer["mixer"]
        h = rnd(around_zero_norm(x, w[p + "norm1"], eps))
        if layer["type"] == "latent_attention":
            j = c.get("kv_from")
            if j is None:
                j = i
                rows[i] = latent_rows(h, w, p + "mix.", c, eps, rnd)
            x = x + m * latent_attention(h, w, p + "mix.", c, rows[j], rnd)
        elif layer["type"] == "retention":
            x = x + m * retention(h, w, p + "mix.", c, eps, rnd)
        else:
            raise ValueError(f"layer type {layer['type']!r}")
        mlp = layer.get("mlp")
        if mlp is not None:
            h = rnd(around_zero_norm(x, w[p + "norm2"], eps))
            if mlp["kind"] == "dense":
                x = x + m * squared_relu_feed_forward(h, w, p + "mlp.", rnd)
            else:
                x = x + m * table_experts(h, w, p + "mlp.", mlp, tokens, rnd)
        if layers_out is not None:
            layers_out.append(x.clone())
    x = rnd(around_zero_norm(x, w["final.norm"], eps))
    return (x @ w["head"].T) * float(cfg["logit_scale"])
