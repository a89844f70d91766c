"""One mechanism of the Gikarax design at a time: a model of one or two layers in which everything else
is quiet, with weights and a prompt made so that a fault shows (a token whose key takes a large share of a
later query's weight from the first position, from both sides of a page's border, just inside and just
outside a window; scores beyond the soft cap; scores near the sink's; a write to a recurrent state that is
read hundreds of tokens later), run through the engine's step function under every cutting, against the
plain implementation.  Each case also checks that it WOULD show the fault: the plain implementation with a
constant or a function changed, or with the far token taken away, moves the probed rows by far more than
the tolerance.  Used on the CPU (kernel wrappers replaced by their PyTorch restatements) and on the GPU."""

from __future__ import annotations

import copy
import math

import torch

from tests import gikarax_util as gu
from tests import plain_gikarax as pg

QUERY, MARKS = 0, (1, 2, 3, 4, 5, 6)       # token ids 0..7 are the marked ones
CLOSE_CALL = 0.12      # a bfloat16 engine may choose another expert where logits are this close


def row_errors(got, want):
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt()


def following(choices, gaps=None):
    """A router for the plain implementation that takes given choices ([experts per token] in the order the
    feed-forwards run), weighted by the rule; ``gaps`` receives how far each token's worst choice lies
    below the rule's last one."""
    left_over = list(choices)

    def choose(h, w, p, top):
        logits = h @ w[p + "router"].T
        ids = left_over.pop(0)
        mine = logits.gather(1, ids)
        if gaps is not None:
            gaps.append(torch.topk(logits, top, dim=-1).values[:, -1] - mine.min(-1).values)
        return ids, torch.softmax(mine, dim=-1)
    return choose


def compare(model_dir, reqs, dtype, device, page, tail, what, **engine):
    """Every schedule's logits against the plain implementation's.  A bfloat16 engine's router sees rounded
    inputs and may decide a close call the other way, which changes everything behind it; so its choices
    are recorded, checked to be the rule's own up to CLOSE_CALL, and the plain implementation follows them.
    Returns (config, weights, the plain logits, the float32 tolerance per request)."""
    cfg, w = pg.read_model_dir(model_dir)
    exact = [pg.forward(cfg, w, r) for r in reqs]
    moe_runs = sum(cfg["layers"][i].get("mlp") is not None for i, _ in pg.layer_runs(cfg))
    lens = [len(r) for r in reqs]
    for name, steps in gu.schedules(lens, tail).items():
        routes = {} if dtype == "bfloat16" and moe_runs else None
        if routes is not None:
            engine = dict(engine, cuda_graphs=False)      # a replayed graph does not show its router's choices
        runner = gu.runner_for(model_dir, dtype, device, page, lens, **engine)
        got = gu.replay(runner, reqs, steps, routes)
        for i, (g, r) in enumerate(zip(got, reqs)):
            e = exact[i]
            if dtype == "float32":
                bound = 1e-4 * float(e.std())
            elif routes is None:
                stored = pg.forward(cfg, w, r, rnd=pg.as_stored_bf16)
                bound = max(3.0 * float(row_errors(stored, e).max()), 2e-2 * float(e.std()))
            else:
                chosen, gaps = [routes[i][k] for k in range(moe_runs)], []
                e = pg.forward(cfg, w, r, choose=following(chosen, gaps))
                for run, gap in enumerate(gaps):
                    assert float(gap.max()) <= CLOSE_CALL, \
                        f"{what} ({dtype}, {name}): request {i}, feed-forward run {run}, position {int(gap.argmax())}: " \
                        f"the engine chose experts whose logits are {float(gap.max()):.3g} from the rule's choice"
                stored = pg.forward(cfg, w, r, rnd=pg.as_stored_bf16, choose=following(chosen))
                bound = max(3.0 * float(row_errors(stored, e).max()), 2e-2 * float(e.std()))
            err = row_errors(g, e)
            worst = int(err.argmax())
            assert float(err[worst]) <= bound, \
                f"{what} ({dtype}, {name}): request {i} position {worst} of {len(e)}: {float(err[worst]):.4g} " \
                f"exceeds {bound:.4g}"
    return cfg, w, exact, [1e-4 * float(e.std()) for e in exact]


def shows(cfg, w, req, exact, bound, rows, what, change_cfg=None, change_req=None, change_w=None, swap=None, factor=30.0):
    """The plain implementation with the change applied moves the probed rows by ``factor`` times the
    float32 engine's tolerance (the bfloat16 engine runs the same case at its own tolerance).  ``swap``: (name,
    function): a function of the plain implementation replaced while it runs."""
    cfg2, req2, w2 = copy.deepcopy(cfg), list(req), dict(w)
    if change_cfg is not None:
        change_cfg(cfg2)
    if change_req is not None:
        change_req(req2)
    if change_w is not None:
        change_w(w2)
    real = None if swap is None else getattr(pg, swap[0])
    try:
        if swap is not None:
            setattr(pg, *swap)
        moved = row_errors(pg.forward(cfg2, w2, req2)[rows], exact[rows])
    finally:
        if swap is not None:
            setattr(pg, swap[0], real)
    assert float(moved.max()) > factor * bound, \
        f"{what}: the case would not show it (rows move by {float(moved.max()):.3g}, tolerance {bound:.3g})"


def filler_tokens(vocab, n, seed):
    g = torch.Generator().manual_seed(seed)
    return (torch.randint(8, vocab, (n,), generator=g)).tolist()


def unmark_at(at):
    def change(r):
        r[at] = 50
    return change


def mark_embeddings(t, size=6.0):
    """Hidden channel 0 marks a key, channel 1 a query, channels 2.. tell the marked keys' values apart; the
    other tokens have nothing there."""
    e = t["embed"]
    e[:, :8] = 0.0
    e[list(MARKS), 0] = size
    e[QUERY, 1] = size
    for j, m in enumerate(MARKS):
        e[m, 2 + j] = 8.0


QUIET_LEFT = gu.left(1, 1, 8, 8, (100.0, 8))
QUIET_RIGHT = gu.right(1, 8, 8, 4.0, 2)


# ---- attention with a window: keys at its edges, page borders, cap, sink, gate, rotation ---------------

def window_case(tmp, dtype, device, heads, kv_heads, dim, vdim, window, rot, page, scaling=None, softcap=None, n=330,
                seed=1, loop=None):
    layer = gu.attention(heads, kv_heads, dim, vdim, window, (5000.0, rot), scaling=scaling, softcap=softcap,
                         scale=1.5 / math.sqrt(dim))
    config = gu.model([layer], 97, 48, loop=loop)

    def edit(t):
        mark_embeddings(t)
        direction = torch.ones(dim)
        if 0 < rot < dim:
            direction[:rot] = 0.0                 # where it can, outside the rotated part
        elif rot:
            direction = torch.zeros(dim)          # else on the pairs that turn slowest
            direction[rot // 2 - 2:rot // 2] = math.sqrt(dim / 2.0)
        t["l0.mix.k"][:, 0] = direction.repeat(kv_heads)
        t["l0.mix.q"][:, 1] = direction.repeat(heads)
        t["l0.mix.k"].mul_(0.7)

    d = gu.write_model(config, seed, tmp, edit)
    toks = filler_tokens(97, n, seed)
    last = n - 1
    # seen from the last three queries: the window's oldest key of each, the one right outside, others far inside
    inside, outside = last - window + 1, last - window
    places = {p: m for p, m in ((0, 1), (last - 5, 4), (inside, 2), (outside, 3)) if 0 <= p < last - 2}
    for p, m in places.items():
        toks[p] = m
    toks[last - 2:] = [QUERY] * 3
    other = filler_tokens(97, 37, seed + 1)
    other[3], other[-1] = 6, QUERY
    reqs = [toks, other, filler_tokens(97, 2 * page + 1, seed + 2)]
    cfg, w, exact, bounds = compare(d, reqs, dtype, device, page, tail=40, what="attention")
    every = list(range(n))
    att = lambda c: c["layers"][0]["mixer"]
    looped = loop is not None and loop[2] > 1
    if inside in places and window > 6:
        # (the last query sees it; the one behind the window's edge is seen by the query before)
        shows(cfg, w, toks, exact[0], bounds[0], [last], "the window's oldest key lost", change_req=unmark_at(inside))
        shows(cfg, w, toks, exact[0], bounds[0], [last], "a window one token shorter",
              change_cfg=lambda c: att(c)["mask"].update(size=window - 1))
    if outside in places:
        shows(cfg, w, toks, exact[0], bounds[0], [last], "a window one token longer",
              change_cfg=lambda c: att(c)["mask"].update(size=window + 1))
    shows(cfg, w, toks, exact[0], bounds[0], every, "no sink",
          swap=("softmax_with_sink", lambda s, seen, sink, real=pg.softmax_with_sink: real(s, seen, False)))
    if softcap is not None:
        shows(cfg, w, toks, exact[0], bounds[0], every, "no soft cap", change_cfg=lambda c: att(c).update(softcap=None))
        shows(cfg, w, toks, exact[0], bounds[0], every, "another soft cap",
              change_cfg=lambda c: att(c).update(softcap=1.2 * softcap))

    def same_gate(w2):
        w2["l0.mix.g"] = w2["l0.mix.g"].mean(0, keepdim=True).expand(heads, -1)
    if heads > 1:
        shows(cfg, w, toks, exact[0], bounds[0], every, "one gate for all heads", change_w=same_gate)
    shows(cfg, w, toks, exact[0], bounds[0], every, "no norm of the queries",
          swap=("rms_norm", lambda x, weight, eps: x * weight))
    if window > 1 and rot:
        shows(cfg, w, toks, exact[0], bounds[0], every, "another base",
              change_cfg=lambda c: att(c)["rot"].update(base=900.0), factor=10.0)
        if scaling is not None:
            shows(cfg, w, toks, exact[0], bounds[0], every, "plain frequencies",
                  change_cfg=lambda c: att(c)["rot"].pop("scaling"), factor=10.0)
    if looped:
        shows(cfg, w, toks, exact[0], bounds[0], every, "a pass less", change_cfg=lambda c: c["loop"].update(times=loop[2] - 1))


# ---- the loop's entry ------------------------------------------------------------------------------------

def loop_case(tmp, dtype, device, loop, page=16, seed=9):
    layers = [gu.attention(2, 1, 16, 16, 20, (1000.0, 8)), gu.latent(2, 16, 16, 24, 16),
              gu.parallel(gu.left(2, 1, 16, 16, (1000.0, 8)), gu.right(2, 16, 16, 4.0, 4)),
              gu.attention(2, 2, 16, 16, 9, (1000.0, 8))]
    d = gu.write_model(gu.model(layers, 97, 48, loop=loop), seed, tmp)
    reqs = gu.requests(97, [90, 33, 2], seed)
    cfg, w, exact, bounds = compare(d, reqs, dtype, device, page, tail=25, what=f"loop {loop}")
    every = list(range(90))
    if loop is None or loop[0] == loop[1]:
        return

    def no_start(w2):
        m = w2["loop.in"].clone()
        m[:, 48:] = 0.0
        w2["loop.in"] = m

    def other_order(w2):
        w2["loop.in"] = torch.cat([w2["loop.in"][:, 48:], w2["loop.in"][:, :48]], dim=1)
    shows(cfg, w, reqs[0], exact[0], bounds[0], every, "the embedding's half lost", change_w=no_start)
    if loop[0] > 0 or loop[2] > 1:
        shows(cfg, w, reqs[0], exact[0], bounds[0], every, "the halves in the other order", change_w=other_order)
        shows(cfg, w, reqs[0], exact[0], bounds[0], every, "another number of passes",
              change_cfg=lambda c: c["loop"].update(times=loop[2] + 1))
    first_only = pg.layer_runs
    if loop[2] > 1:
        def once(cfg_):
            seen = set()
            return [(i, e and not (i in seen or seen.add(i))) for i, e in first_only(cfg_)]
        shows(cfg, w, reqs[0], exact[0], bounds[0], every, "an entry in front of the first pass only",
              swap=("layer_runs", once))
    shows(cfg, w, reqs[0], exact[0], bounds[0], every, "a norm that keeps the mean",
          swap=("layer_norm", pg.rms_norm))


# ---- the left half: biases, blended frequencies, far keys ----------------------------------------------

def left_case(tmp, dtype, device, heads, kv_heads, dim, vdim, rot, page, scaling=None, n=330, seed=3):
    half = gu.left(heads, kv_heads, dim, vdim, (5000.0, rot), scaling=scaling, scale=2.4 / dim)
    config = gu.model([gu.parallel(half, QUIET_RIGHT)], 97, 48)

    def edit(t):
        mark_embeddings(t)
        direction = torch.ones(dim)
        if 0 < rot < dim:
            direction[:rot] = 0.0                 # where it can, outside the rotated part
        elif rot:
            direction = torch.zeros(dim)          # else on the pairs that turn slowest
            direction[rot // 2 - 2:rot // 2] = math.sqrt(dim / 2.0)
        for x, ch, hh in (("k", 0, kv_heads), ("q", 1, heads)):
            t[f"l0.mix.left.{x}"].mul_(0.3)
            t[f"l0.mix.left.{x}"][:, ch] = 0.8 * direction.repeat(hh)
        t["l0.mix.right.out"].zero_()             # the other branch is silent

    d = gu.write_model(config, seed, tmp, edit)
    toks = filler_tokens(97, n, seed)
    last = n - 1
    # marked keys: the first token, both sides of a page's border far back, the middle, right before the queries
    places = {0: 1, 2 * page - 1: 2, 2 * page: 3, n // 2: 4, last - 4: 5}
    for p, m in places.items():
        toks[p] = m
    toks[last - 2:] = [QUERY] * 3
    other = filler_tokens(97, 37, seed + 1)
    other[3], other[-1] = 6, QUERY
    reqs = [toks, other, filler_tokens(97, 2 * page + 1, seed + 2)]
    cfg, w, exact, bounds = compare(d, reqs, dtype, device, page, tail=40, what="attention with biases")
    rows, every = list(range(last - 2, n)), list(range(n))
    att = lambda c: c["layers"][0]["mixer"]["left"]
    for p in (0, 2 * page - 1, 2 * page, n // 2):
        shows(cfg, w, toks, exact[0], bounds[0], rows, f"the far key at {p} lost", change_req=unmark_at(p),
              factor=30.0 if rot < dim else 8.0)

    def without(x):
        def change(w2):
            w2[f"l0.mix.left.{x}.b"] = torch.zeros_like(w2[f"l0.mix.left.{x}.b"])
        return change
    for x in ("q", "v", "o") + (("k",) if rot else ()):       # (a key bias without a rotation: the softmax drops it)
        shows(cfg, w, toks, exact[0], bounds[0], every, f"no bias of {x}", change_w=without(x), factor=10.0)

    def swapped_norms(w2):
        w2["l0.mix.left.out"] = torch.ones_like(w2["l0.mix.left.out"])
    shows(cfg, w, toks, exact[0], bounds[0], every, "no weight of the branch's norm", change_w=swapped_norms)
    if rot:
        shows(cfg, w, toks, exact[0], bounds[0], every, "another base", change_cfg=lambda c: att(c)["rot"].update(base=900.0),
              factor=10.0)
    if scaling is not None:
        shows(cfg, w, toks, exact[0], bounds[0], every, "plain frequencies",
              change_cfg=lambda c: att(c)["rot"].pop("scaling"), factor=10.0)
        shows(cfg, w, toks, exact[0], bounds[0], every, "no factor on cosine and sine",
              swap=("blended_frequencies", lambda *a, real=pg.blended_frequencies: (real(*a)[0], 1.0)), factor=10.0)


# ---- the right half: gated linear attention ------------------------------------------------------------

def gated_linear_case(tmp, dtype, device, heads, dim, vdim, tau, rank, page=16, n=330, seed=4):
    config = gu.model([gu.parallel(QUIET_LEFT, gu.right(heads, dim, vdim, tau, rank))], 97, 48)

    def edit(t):
        # a marked token writes a large value under a key that only the marked query, far behind, asks for, on
        # the half of the channels that forgets slowly; the other half forgets fast
        mark_embeddings(t, 9.0)
        p = "l0.mix.right."
        slow = torch.zeros(dim)
        slow[dim // 2:] = 1.0
        for x, ch in (("q", 1), ("k", 0)):
            t[p + x].mul_(0.3)
            t[p + x].view(heads, dim, -1)[:, :, ch] = slow
        t[p + "v"][:, 2] = 2.0
        t[p + "a2"].mul_(0.7)
        t[p + "a2"].view(heads, dim, rank)[:, dim // 2:] *= 0.1
        t[p + "a2.b"].view(heads, dim)[:] = torch.where(slow > 0, 6.0 - math.log(tau), 0.5)
        t["l0.mix.left.out"].zero_()              # the other branch is silent

    d = gu.write_model(config, seed, tmp, edit)
    toks = filler_tokens(97, n, seed)
    toks[2] = MARKS[0]
    toks[n - 2:] = [QUERY] * 2
    # (lengths at and beside a chunk of 64 tokens and a run of 16)
    reqs = [toks] + [filler_tokens(97, m, seed + i) for i, m in enumerate((64, 17, 3, 65, 128, 63, 16))]
    cfg, w, exact, bounds = compare(d, reqs, dtype, device, page, tail=100, what="gated linear attention")
    every = list(range(n))
    mix = lambda c: c["layers"][0]["mixer"]["right"]
    shows(cfg, w, toks, exact[0], bounds[0], [n - 2, n - 1], "a write lost from the state", change_req=unmark_at(2), factor=15.0)
    shows(cfg, w, toks, exact[0], bounds[0], every, "another tau", change_cfg=lambda c: mix(c).update(tau=1.1 * tau))
    shows(cfg, w, toks, exact[0], bounds[0], every, "another eps", change_cfg=lambda c: c["norm"].update(eps=3e-3), factor=5.0)

    def one_decay(hh, ww, p, tau_, real=pg.channel_decays):
        a = real(hh, ww, p, tau_)
        return a.reshape(a.shape[0], heads, dim).mean(-1, keepdim=True).expand(-1, -1, dim).reshape(a.shape)
    shows(cfg, w, toks, exact[0], bounds[0], every, "one decay for all channels", swap=("channel_decays", one_decay))

    def values_decay(q, k, v, alpha, real=pg.gated_linear_recurrence):
        return real(q, k, v, alpha.roll(1, dims=0))
    shows(cfg, w, toks, exact[0], bounds[0], every, "the decay of the token before", swap=("gated_linear_recurrence", values_decay))

    def no_norm_weight(w2):
        w2["l0.mix.right.norm"] = torch.ones_like(w2["l0.mix.right.norm"])
    if vdim > 1:
        shows(cfg, w, toks, exact[0], bounds[0], every, "no weight of the heads' norm", change_w=no_norm_weight)


# ---- latent attention ------------------------------------------------------------------------------------

def latent_case(tmp, dtype, device, heads, dim, vdim, kv_rank, q_rank, page, n=330, seed=5):
    config = gu.model([gu.latent(heads, dim, vdim, kv_rank, q_rank, scale=2.0 / dim)], 97, 48)

    def edit(t):
        # through element 0 of both latents a marked query and a marked key meet on one direction of every head;
        # latent elements 1..6 carry the marked keys' values
        mark_embeddings(t)
        p = "l0.mix."
        t[p + "dkv"][:8] *= 0.05
        t[p + "dkv"][0, 0] = 1.5
        for j in range(6):
            t[p + "dkv"][1 + j, 2 + j] = 1.5
        t[p + "dq"].mul_(0.3)
        t[p + "dq"][0, 1] = 1.5
        t[p + "uk"].mul_(0.2)
        t[p + "uk"][:, 0] = math.sqrt(24.0 / kv_rank)      # (an element of a normed latent grows with its size)
        t[p + "uq"].mul_(0.3)
        t[p + "uq"][:, 0] = 0.6 * math.sqrt(12.0 / q_rank)

    d = gu.write_model(config, seed, tmp, edit)
    toks = filler_tokens(97, n, seed)
    last = n - 1
    for p, m in {0: 1, 2 * page - 1: 2, 2 * page: 3, n // 2: 4, last - 4: 5}.items():
        toks[p] = m
    toks[last - 2:] = [QUERY] * 3
    other = filler_tokens(97, 37, seed + 1)
    other[3], other[-1] = 6, QUERY
    reqs = [toks, other, filler_tokens(97, 2 * page + 1, seed + 2)]
    cfg, w, exact, bounds = compare(d, reqs, dtype, device, page, tail=40, what="latent attention")
    rows, every = list(range(last - 2, n)), list(range(n))
    for at in (0, 2 * page - 1, 2 * page, n // 2):
        shows(cfg, w, toks, exact[0], bounds[0], rows, f"the far key at {at} lost", change_req=unmark_at(at))

    def ones(name):
        def change(w2):
            w2[name] = torch.ones_like(w2[name])
        return change

    def no_gate(w2):
        w2["l0.mix.g"] = torch.zeros_like(w2["l0.mix.g"])

    def gate_by_head(w2):
        g = w2["l0.mix.g"].reshape(heads, vdim, -1)
        w2["l0.mix.g"] = g.mean(1, keepdim=True).expand(-1, vdim, -1).reshape(heads * vdim, -1)
    shows(cfg, w, toks, exact[0], bounds[0], every, "no weight of the query latent's norm", change_w=ones("l0.mix.dq.norm"))
    shows(cfg, w, toks, exact[0], bounds[0], every, "no weight of the latent's norm", change_w=ones("l0.mix.dkv.norm"))
    shows(cfg, w, toks, exact[0], bounds[0], every, "no gate", change_w=no_gate)
    if vdim > 1:
        shows(cfg, w, toks, exact[0], bounds[0], every, "one gate number per head", change_w=gate_by_head)
    shows(cfg, w, toks, exact[0], bounds[0], every, "another scale",
          change_cfg=lambda c: c["layers"][0]["mixer"].update(scale=2.5 / dim))


# ---- experts ---------------------------------------------------------------------------------------------

def experts_case(tmp, dtype, device, experts, top, ff, page=16, seed=6):
    config = gu.model([gu.attention(1, 1, 8, 8, 2, (100.0, 8), mlp=gu.moe(experts, top, ff))], 97, 48)

    def edit(t):
        t["l0.mix.o"].mul_(0.05)                    # the mixer nearly silent: the feed-forward is what is left

    d = gu.write_model(config, seed, tmp, edit)
    reqs = [filler_tokens(97, n, seed + i) for i, n in enumerate((90, 17, 1, 300))]
    cfg, w, exact, bounds = compare(d, reqs, dtype, device, page, tail=20, what="experts")
    rows = list(range(90))
    tanh_gelu = lambda z: 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))
    shows(cfg, w, reqs[0], exact[0], bounds[0], rows, "the tanh form of the gelu", swap=("gelu", tanh_gelu), factor=1.5)
    if 1 < top:
        def softmax_over_all(h, ww, p, k, real=pg.chosen_experts):
            ids, _ = real(h, ww, p, k)
            return ids, torch.softmax(h @ ww[p + "router"].T, dim=-1).gather(1, ids)
        if top < experts:
            shows(cfg, w, reqs[0], exact[0], bounds[0], rows, "weights from all experts", swap=("chosen_experts", softmax_over_all))

        def equal(h, ww, p, k, real=pg.chosen_experts):
            ids, share = real(h, ww, p, k)
            return ids, torch.full_like(share, 1.0 / k)
        shows(cfg, w, reqs[0], exact[0], bounds[0], rows, "equal weights", swap=("chosen_experts", equal))
    if top < experts:
        shows(cfg, w, reqs[0], exact[0], bounds[0], rows, "an expert more",
              change_cfg=lambda c: c["layers"][0]["mlp"]["router"].update(top=top + 1))

    def behind(cfg_, ww, tokens, rnd=pg._keep, layers_out=None, choose=None):      # the experts read the mixer's sum
        eps = float(cfg_["norm"]["eps"])
        x = ww["embed"][torch.as_tensor(list(tokens), dtype=torch.long)]
        x = x + pg.attention(pg.layer_norm(x, ww["l0.norm1"], eps), ww, "l0.mix.", cfg_["layers"][0]["mixer"], eps)
        x = x + pg.mixture(pg.layer_norm(x, ww["l0.norm1"], eps), ww, "l0.mlp.", cfg_["layers"][0]["mlp"])
        return pg.layer_norm(x, ww["final.norm"], eps) @ ww["head"].T
    shows(cfg, w, reqs[0], exact[0], bounds[0], rows, "sublayers one behind the other", swap=("forward", behind), factor=10.0)
