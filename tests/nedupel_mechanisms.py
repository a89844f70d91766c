"""One mechanism of the Nedupel design at a time: a model of one or two layers in which everything
else is quiet, with weights and a prompt made so that a fault shows (a token whose key takes nearly all of
a later query's weight from the first position, from both sides of a page's border far back and from the
middle; a write to a retention state that is read hundreds of tokens later; gates beyond their limits),
run through the engine's step function under every cutting, against the plain implementation.  Each case
also checks that it WOULD show the fault: the plain implementation with the constant changed, or with
the far token taken away, moves the probed rows by far more than the tolerance.  Used on the CPU (kernel
wrappers replaced by their PyTorch restatements) and on the GPU."""

from __future__ import annotations

import copy

import torch

from tests import nedupel_util as nu
from tests import plain_nedupel as pn

QUERY, MARKS = 0, (1, 2, 3, 4, 5, 6)       # token ids 0..7 are the marked ones


def row_errors(got, want):
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt()


def bound_of(cfg, w, req, exact, dtype):
    """What an engine of this type may differ by: float32 1e-4 of the logits' spread; bfloat16 three
    times what storing in bfloat16 alone does to the plain implementation."""
    if dtype == "float32":
        return 1e-4 * float(exact.std())
    stored = pn.forward(cfg, w, req, rnd=pn.as_stored_bf16)
    return max(3.0 * float(row_errors(stored, exact).max()), 2e-2 * float(exact.std()))


def compare(model_dir, reqs, dtype, device, page, tail, what, **engine):
    """Every schedule's logits against the plain implementation's.  Returns (config, weights, the plain
    logits, the float32 tolerance per request)."""
    cfg, w = pn.read_model_dir(model_dir)
    exact = [pn.forward(cfg, w, r) for r in reqs]
    bounds = [bound_of(cfg, w, r, e, dtype) for r, e in zip(reqs, exact)]
    lens = [len(r) for r in reqs]
    for name, steps in nu.schedules(lens, tail).items():
        runner = nu.runner_for(model_dir, dtype, device, page, lens, **engine)
        for i, (g, e, bound) in enumerate(zip(nu.replay(runner, reqs, steps), exact, bounds)):
            err = row_errors(g, e)
            worst = int(err.argmax())
            assert float(err[worst]) <= bound, \
                f"{what} ({dtype}, {name}): request {i} position {worst} of {len(e)}: {float(err[worst]):.4g} " \
                f"exceeds {bound:.4g}"
    return cfg, w, exact, [1e-4 * float(e.std()) for e in exact]


def shows(cfg, w, req, exact, bound, rows, what, change_cfg=None, change_req=None, change_w=None, factor=30.0):
    """The plain implementation with the change applied moves the probed rows by ``factor`` times the
    float32 engine's tolerance (the bfloat16 engine runs the same case at its own tolerance)."""
    cfg2, req2, w2 = copy.deepcopy(cfg), list(req), dict(w)
    if change_cfg is not None:
        change_cfg(cfg2)
    if change_req is not None:
        change_req(req2)
    if change_w is not None:
        change_w(w2)
    moved = row_errors(pn.forward(cfg2, w2, req2)[rows], exact[rows])
    assert float(moved.max()) > factor * bound, \
        f"{what}: the case would not show it (rows move by {float(moved.max()):.3g}, tolerance {bound:.3g})"


def filler_tokens(vocab, n, seed):
    g = torch.Generator().manual_seed(seed)
    return (torch.randint(8, vocab, (n,), generator=g)).tolist()


# ---- latent attention: far keys, page borders, the rotation, rows of another layer -------------------

def latent_case(tmp, dtype, device, heads, dim, rot_dim, vdim, rank, page, scaling=None, shared=False, n=330, seed=1):
    """``shared``: a second layer reads the first one's rows (its own output is all that reaches the
    probed rows from far back: the first layer's output projection is silent)."""
    layers = [nu.latent(heads, dim, rot_dim, vdim, rank, 500.0, scaling=scaling, scale=2.4 / dim)]
    if shared:
        layers.append(nu.latent(heads + 1, dim, rot_dim, vdim, rank, 500.0, scaling=scaling, scale=2.4 / dim, kv_from=0))
    config = nu.model(layers, 97, 48, mult=0.7, embed=1.0)
    reader = len(layers) - 1

    def edit(t):
        # hidden channel 0 marks a key, channel 1 a query; through the latent's element 0 both map onto the
        # same direction of every head's plain part, so a marked key takes most of a marked query's
        # weight; channels 2.. tell the marked keys' values apart (latent elements 1..6)
        e = t["embed"]
        e[:, :8] = 0.0
        e[list(MARKS), 0] = 6.0
        e[QUERY, 1] = 6.0
        for j, m in enumerate(MARKS):
            e[m, 2 + j] = 8.0
        down = t["l0.mix.dkv"]
        down[:8] *= 0.05
        down[0, 0] = 1.5
        for j in range(6):
            down[1 + j, 2 + j] = 1.5
        p = f"l{reader}.mix."
        h = layers[reader]["mixer"]["heads"]
        t[p + "uk"].mul_(0.2)
        t[p + "uk"][:, 0] = 1.0
        t[p + "q"].mul_(0.3)
        t[p + "q"].view(h, dim + rot_dim, -1)[:, :dim, 1] = 0.2
        if shared:
            t["l0.mix.o"].zero_()

    d = nu.write_model(config, seed, tmp, edit)
    toks = filler_tokens(97, n, seed)
    last = n - 1
    # marked keys: the first token, both sides of a page's border far back, the middle, right before the queries
    places = {0: 1, 2 * page - 1: 2, 2 * page: 3, n // 2: 4, last - 4: 5}
    for at, m in places.items():
        toks[at] = m
    toks[last - 2:] = [QUERY] * 3
    other = filler_tokens(97, 37, seed + 1)
    other[3], other[-1] = 6, QUERY
    reqs = [toks, other, filler_tokens(97, 2 * page + 1, seed + 2)]
    cfg, w, exact, bounds = compare(d, reqs, dtype, device, page, tail=40, what="latent attention")
    rows, every = list(range(last - 2, n)), list(range(n))
    for at in (0, 2 * page - 1, 2 * page, n // 2):
        def unmark(r, at=at):
            r[at] = 50
        shows(cfg, w, toks, exact[0], bounds[0], rows, f"the far key at {at} lost", change_req=unmark)

    def rots(c):
        return [layer["mixer"]["rot"] for layer in c["layers"]]
    if scaling is not None:
        shows(cfg, w, toks, exact[0], bounds[0], every, "plain frequencies",
              change_cfg=lambda c: [r.pop("scaling") for r in rots(c)])
        shows(cfg, w, toks, exact[0], bounds[0], every, "another share of the blend",
              change_cfg=lambda c: [r["scaling"].update(slow=r["scaling"]["fast"] * 0.99) for r in rots(c)], factor=10.0)
    shows(cfg, w, toks, exact[0], bounds[0], every, "another base",
          change_cfg=lambda c: [r.update(base=900.0) for r in rots(c)], factor=10.0)


# ---- retention -----------------------------------------------------------------------------------------

def retention_case(tmp, dtype, device, dim, vdim, decay, rot, page=16, n=330, seed=2):
    config = nu.model([nu.retention(dim, vdim, decay, 5000.0, rot)], 97, 48, mult=0.9)
    heads = len(decay)

    def edit(t):
        # a marked token writes a large value under a key that only the marked query, far behind, asks for
        # (where it can, outside the rotated part: a key of low frequency there otherwise)
        e = t["embed"]
        e[:, :8] = 0.0
        e[MARKS[0], 0] = 9.0
        e[QUERY, 1] = 9.0
        e[MARKS[0], 2] = 9.0
        t["l0.mix.q"].mul_(0.3)
        t["l0.mix.k"].mul_(0.3)
        half = rot // 2
        for x, ch in (("q", 1), ("k", 0)):
            m = t[f"l0.mix.{x}"].view(heads, dim, -1)
            if rot < dim:
                m[:, rot:, ch] = 1.0
            else:
                m[:, half // 2:half, ch] = 1.0
        t["l0.mix.v"][:, 2] = 2.0

    d = nu.write_model(config, seed, tmp, edit)
    toks = filler_tokens(97, n, seed)
    toks[2] = MARKS[0]
    toks[n - 2:] = [QUERY] * 2
    # (lengths at and beside a chunk of 64 tokens)
    reqs = [toks] + [filler_tokens(97, m, seed + i) for i, m in enumerate((64, 29, 3, 65, 128, 63))]
    cfg, w, exact, bounds = compare(d, reqs, dtype, device, page, tail=100, what="retention")
    mix = lambda c: c["layers"][0]["mixer"]
    every = list(range(n))

    def unmark(r):
        r[2] = 50
    shows(cfg, w, toks, exact[0], bounds[0], [n - 2, n - 1], "a write lost from the state", change_req=unmark, factor=15.0)
    shows(cfg, w, toks, exact[0], bounds[0], every, "another decay",
          change_cfg=lambda c: mix(c).update(decay=[0.98 * x for x in decay]))
    # (k's factor only meets the norm's eps, which the first tokens show)
    shows(cfg, w, toks, exact[0], bounds[0], every, "another eps", change_cfg=lambda c: c["norm"].update(eps=3e-3), factor=5.0)
    if rot:
        shows(cfg, w, toks, exact[0], bounds[0], every, "another base",
              change_cfg=lambda c: mix(c)["rot"].update(base=100.0), factor=10.0)
    if rot < dim:
        shows(cfg, w, toks, exact[0], bounds[0], every, "a wider rotation",
              change_cfg=lambda c: mix(c)["rot"].update(dims=dim // 2 * 2), factor=10.0)


# ---- feed-forwards ---------------------------------------------------------------------------------------

def _quiet_mixer_model(mlp):
    return nu.model([nu.retention(8, 8, (0.9,), 100.0, 8, mlp=mlp)], 97, 48, mult=0.6)


def experts_case(tmp, dtype, device, experts, top, ff, limit, page=16, seed=4):
    def edit(t):
        t["l0.mix.o"].mul_(0.05)                    # the mixer nearly silent: the feed-forward reads the embedding

    d = nu.write_model(_quiet_mixer_model(nu.moe(experts, top, ff, limit)), seed, tmp, edit)
    reqs = [filler_tokens(97, n, seed + i) for i, n in enumerate((90, 17, 1, 300))]
    cfg, w, exact, bounds = compare(d, reqs, dtype, device, page, tail=20, what="experts of a table")
    rows = list(range(90))
    shows(cfg, w, reqs[0], exact[0], bounds[0], rows, "another limit",
          change_cfg=lambda c: c["layers"][0]["mlp"]["expert"].update(limit=1.1 * limit), factor=20.0)
    if top < experts:
        def next_expert(w2):
            w2["l0.mlp.table"] = (w2["l0.mlp.table"] + 1) % experts
        shows(cfg, w, reqs[0], exact[0], bounds[0], rows, "another table", change_w=next_expert)


def dense_case(tmp, dtype, device, ff, page=16, seed=5):
    def edit(t):
        t["l0.mix.o"].mul_(0.05)

    d = nu.write_model(_quiet_mixer_model(nu.dense(ff)), seed, tmp, edit)
    reqs = [filler_tokens(97, n, seed + i) for i, n in enumerate((90, 17, 1, 300))]
    cfg, w, exact, bounds = compare(d, reqs, dtype, device, page, tail=20, what="squared relu")

    def double(w2):                                 # twice the input: four times the square
        w2["l0.mlp.up"], w2["l0.mlp.down"] = 2.0 * w2["l0.mlp.up"], 0.5 * w2["l0.mlp.down"]
    shows(cfg, w, reqs[0], exact[0], bounds[0], list(range(90)), "not a square", change_w=double)
    shows(cfg, w, reqs[0], exact[0], bounds[0], list(range(90)), "another factor on the branches",
          change_cfg=lambda c: c.update(residual_mult=0.62))
