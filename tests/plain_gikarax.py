"""A plain, slow implementation of the Gikarax design: whole sequences, no cache, no batches,
float64 by default, one function per mechanism, written from the design's equations.  It shares
no code with the package; the tests compare the package with it.

Notation: n tokens, width W.  ``w`` maps tensor names to tensors, ``p`` is a part's prefix
("l3.mix." and the like), ``c`` the part's entry of config.json.  ``rnd`` rounds what a
bfloat16 engine stores (a yardstick for its tests); by default nothing is rounded.

The stream starts as embed[token].  A layer is x <- x + (mixer(h) + ff(h)) with ONE layer norm
h = norm1(x).  A run of layers is repeated with the same weights; in front of each pass the stream
becomes loop.in [x; x0], x0 the embedding's output.  Mixers: "attention" (window, capped scores, a
sink of score 0, one gate number per head), "parallel" (attention with biases beside gated linear
attention, each normed over the width, halved and added) and "latent_attention" (keys and values
from a small latent per token, queries through a latent too, no positions, an element-wise gate).
The feed-forward is a mixture of ungated experts.
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
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16}
    out = {}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        a, b = meta["data_offsets"]
        t = torch.frombuffer(bytearray(data[a:b]), dtype=kinds[meta["dtype"]]).reshape(meta["shape"])
        out[name] = t.to(dtype)
    return cfg, out


def _keep(x):
    return x


def as_stored_bf16(x):
    return x.to(torch.bfloat16).to(x.dtype)


# ---- small functions -------------------------------------------------------------------------

def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def layer_norm(x, weight, eps):
    centred = x - x.mean(-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(-1, keepdim=True) + eps) * weight


def silu(z):
    return z * torch.sigmoid(z)


def gelu(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


# ---- rotations ---------------------------------------------------------------------------------

def plain_frequencies(dims, base):
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def stretched_frequencies(dims, base, scaling):
    """Long wavelengths stretched: short ones stay, long ones turn ``factor`` times slower, a blend between."""
    freqs = plain_frequencies(dims, base)
    if scaling is None:
        return freqs
    factor, low, high, original = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
    out = []
    for f in freqs:
        length = 2.0 * math.pi / f
        if length < original / high:
            out.append(f)
        elif length > original / low:
            out.append(f / factor)
        else:
            s = (original / length - low) / (high - low)
            out.append((1.0 - s) * f / factor + s * f)
    return out


def blended_frequencies(dims, base, scaling):
    """(frequencies, factor on cosine and sine): blended by the pair's index between the pair that turns
    ``fast`` times over ``original`` positions and the one that turns ``slow`` times."""
    freqs = plain_frequencies(dims, base)
    if scaling is None:
        return freqs, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def index_of(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(float(scaling["fast"]))), 0)
    hi = min(math.ceil(index_of(float(scaling["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * r + f * (1.0 - r))
    return out, 0.1 * math.log(factor) + 1.0


def rotate_halves(x, positions, freqs, size=1.0):
    """x [n, heads, D]: element i turns with element i + pairs by position * f_i; elements from 2 pairs
    on pass.  ``size`` multiplies cosine and sine."""
    half = len(freqs)
    a = positions.to(x.dtype)[:, None] * torch.tensor(freqs, dtype=x.dtype)[None, :]
    cos, sin = size * torch.cos(a)[:, None, :], size * torch.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., 2 * half:]], dim=-1)


# ---- attention over given q, k, v ------------------------------------------------------------------

def visible(n, window):
    """[n, n] bool: query i (row) sees key j (column)."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    seen = j <= i
    return seen if window is None else seen & (i - j < window)


def capped(scores, cap):
    return scores if cap is None else cap * torch.tanh(scores / cap)


def softmax_with_sink(scores, seen, sink):
    """Softmax over the keys seen; ``sink``: one more term of score 0 in the denominator."""
    scores = scores.masked_fill(~seen, -math.inf)
    top = scores.max(-1, keepdim=True).values
    if sink:
        top = top.clamp(min=0.0)
    p = torch.exp(scores - top)
    den = p.sum(-1, keepdim=True)
    return p / (den + torch.exp(-top) if sink else den)


def attend(q, k, v, scale, window=None, cap=None, sink=False):
    """q [n, H, D], k [n, G, D], v [n, G, E] -> [n, H, E]; query head h reads key head h // (H / G)."""
    n, heads, _ = q.shape
    per = heads // k.shape[1]
    seen = visible(n, window)
    out = torch.zeros(n, heads, v.shape[-1], dtype=q.dtype)
    for h in range(heads):
        s = capped(q[:, h] @ k[:, h // per].T * scale, cap)
        out[:, h] = softmax_with_sink(s, seen, sink) @ v[:, h // per]
    return out


# ---- mixer "attention" -----------------------------------------------------------------------------

def attention(h, w, p, c, eps, rnd=_keep):
    n, heads, groups, d, e = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = rms_norm(rnd(h @ w[p + "q"].T).reshape(n, heads, d), w[p + "q.norm"], eps)
    k = rms_norm(rnd(h @ w[p + "k"].T).reshape(n, groups, d), w[p + "k.norm"], eps)
    v = rnd(h @ w[p + "v"].T).reshape(n, groups, e)
    rot = c.get("rot")
    if rot is not None:
        freqs = stretched_frequencies(rot["dims"], float(rot["base"]), rot.get("scaling"))
        q, k = (rotate_halves(x, torch.arange(n), freqs) for x in (q, k))
    cap = c.get("softcap")
    window = None if c.get("mask") is None else int(c["mask"]["size"])
    o = rnd(attend(rnd(q), rnd(k), v, float(c["scale"]), window, None if cap is None else float(cap), sink=True))
    o = rnd(o * torch.sigmoid(rnd(h @ w[p + "g"].T))[:, :, None])
    return rnd(o.reshape(n, heads * e) @ w[p + "o"].T)


# ---- mixer "parallel" ------------------------------------------------------------------------------

def biased_attention(h, w, p, c, rnd=_keep):
    n, heads, groups, d, e = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = rnd(h @ w[p + "q"].T + w[p + "q.b"]).reshape(n, heads, d)
    k = rnd(h @ w[p + "k"].T + w[p + "k.b"]).reshape(n, groups, d)
    v = rnd(h @ w[p + "v"].T + w[p + "v.b"]).reshape(n, groups, e)
    rot = c.get("rot")
    if rot is not None:
        freqs, size = blended_frequencies(rot["dims"], float(rot["base"]), rot.get("scaling"))
        q, k = (rotate_halves(x, torch.arange(n), freqs, size) for x in (q, k))
    o = rnd(attend(rnd(q), rnd(k), v, float(c["scale"])))
    return rnd(o.reshape(n, heads * e) @ w[p + "o"].T + w[p + "o.b"])


def gated_linear_recurrence(q, k, v, alpha):
    """q, k, alpha [n, H, D], v [n, H, E].  Per head from S = 0 [D, E]: S <- diag(alpha) S + k v^T; o = S^T q."""
    n, heads, d = q.shape
    s = torch.zeros(heads, d, v.shape[-1], dtype=q.dtype)
    out = torch.zeros(n, heads, v.shape[-1], dtype=q.dtype)
    for t in range(n):
        s = alpha[t][:, :, None] * s + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (s * q[t][:, :, None]).sum(1)
    return out


def channel_decays(h, w, p, tau):
    """[n, H D]: sigmoid(z)^(1/tau), z through a low-rank map with a bias at its end."""
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    return torch.exp(torch.nn.functional.logsigmoid(z) / tau)


def gated_linear_attention(h, w, p, c, eps, rnd=_keep):
    n, heads, d, e = h.shape[0], c["heads"], c["dim"], c["vdim"]
    q = rnd(h @ w[p + "q"].T).reshape(n, heads, d) * d ** -0.5
    k = rnd(h @ w[p + "k"].T).reshape(n, heads, d)
    v = rnd(h @ w[p + "v"].T).reshape(n, heads, e)
    alpha = channel_decays(h, w, p, float(c["tau"])).reshape(n, heads, d)
    o = rms_norm(gated_linear_recurrence(q, k, v, alpha), w[p + "norm"], eps).reshape(n, heads * e)
    return rnd(rnd(o * silu(rnd(h @ w[p + "g"].T))) @ w[p + "o"].T)


def side_by_side(h, w, p, c, eps, rnd=_keep):
    left = biased_attention(h, w, p + "left.", c["left"], rnd)
    right = gated_linear_attention(h, w, p + "right.", c["right"], eps, rnd)
    return 0.5 * (rms_norm(left, w[p + "left.out"], eps) + rms_norm(right, w[p + "right.out"], eps))


# ---- mixer "latent_attention" ---------------------------------------------------------------------

def latent_attention(h, w, p, c, eps, rnd=_keep):
    n, heads, d, e = h.shape[0], c["heads"], c["dim"], c["vdim"]
    q_latent = rnd(rms_norm(rnd(h @ w[p + "dq"].T), w[p + "dq.norm"], eps))
    q = rnd(q_latent @ w[p + "uq"].T).reshape(n, heads, d)
    latent = rnd(rms_norm(rnd(h @ w[p + "dkv"].T), w[p + "dkv.norm"], eps))
    k = rnd(latent @ w[p + "uk"].T).reshape(n, heads, d)
    v = rnd(latent @ w[p + "uv"].T).reshape(n, heads, e)
    o = rnd(attend(q, k, v, float(c["scale"]))).reshape(n, heads * e)
    return rnd(rnd(o * torch.sigmoid(rnd(h @ w[p + "g"].T))) @ w[p + "o"].T)


# ---- feed-forward ---------------------------------------------------------------------------------

def chosen_experts(h, w, p, top):
    """([n, top] experts, [n, top] weights): the largest logits, weighted by the softmax over them alone."""
    logits = h @ w[p + "router"].T
    best = torch.topk(logits, top, dim=-1)
    return best.indices, torch.softmax(best.values, dim=-1)


def expert(h, w, p, rnd=_keep):
    return rnd(rnd(gelu(rnd(h @ w[p + "up"].T))) @ w[p + "down"].T)


def mixture(h, w, p, c, rnd=_keep, choose=None):
    ids, weights = (choose or chosen_experts)(h, w, p, c["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(c["router"]["experts"]):
        share = (weights * (ids == e)).sum(-1)
        rows = (ids == e).any(-1)
        if bool(rows.any()):
            out[rows] += share[rows, None] * expert(h[rows], w, f"{p}e{e}.", rnd)
    return out


# ---- the model ------------------------------------------------------------------------------------

def layer_runs(cfg):
    """(layer, whether a pass of the loop starts in front of it) in the order the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if loop is None:
        return [(i, False) for i in range(n)]
    start, stop = loop["start"], loop["stop"]
    runs = [(i, False) for i in range(start)]
    for _ in range(loop["times"]):
        runs += [(i, i == start) for i in range(start, stop)]
    return runs + [(i, False) for i in range(stop, n)]


def forward(cfg, w, tokens, rnd=_keep, layers_out=None, choose=None):
    """Logits [n, vocab] of one sequence.  ``layers_out``: a list that receives the residual stream
    after every layer run."""
    eps = float(cfg["norm"]["eps"])
    x0 = w["embed"][torch.as_tensor([int(t) for t in tokens], dtype=torch.long)]
    x = x0
    for i, enters in layer_runs(cfg):
        layer = cfg["layers"][i]
        p, c = f"l{i}.", layer["mixer"]
        if enters:
            x = rnd(torch.cat([x, x0], dim=-1)) @ w["loop.in"].T
        h = rnd(layer_norm(x, w[p + "norm1"], eps))
        if layer["type"] == "attention":
            y = attention(h, w, p + "mix.", c, eps, rnd)
        elif layer["type"] == "parallel":
            y = side_by_side(h, w, p + "mix.", c, eps, rnd)
        elif layer["type"] == "latent_attention":
            y = latent_attention(h, w, p + "mix.", c, eps, rnd)
        else:
            raise ValueError(f"layer type {layer['type']!r}")
        if layer.get("mlp") is not None:
            y = y + mixture(h, w, p + "mlp.", layer["mlp"], rnd, choose)
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return rnd(layer_norm(x, w["final.norm"], eps)) @ w["head"].T
