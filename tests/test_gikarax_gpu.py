"""The Gikarax design on the GPU against the plain implementation of ``tests/plain_gikarax.py``: each
mechanism alone (``tests/gikarax_mechanisms.py``), the new kernels alone against their equations, then whole
models under every cutting (whole prompts, the last tokens one by one, portions down to two tokens, mixed
batches in a pool so small that pages and slots are used again), in float32 through ``bin/trace_run`` and in
both types through the step function; with captured graphs; and greedy generation through
``Engine.generate``."""

import copy
import math

import pytest
import torch

from tests import gikarax_mechanisms as gm
from tests import gikarax_util as gu
from tests import plain_gikarax as pg
from tests import replay_util as ru

pytestmark = pytest.mark.gpu

DTYPES = ("float32", "bfloat16")


@pytest.fixture(scope="module")
def model_dirs(tmp_path_factory):
    return {name: gu.write_tiny(name, tmp_path_factory.mktemp(f"gikarax_{name}")) for name in gu.CONFIGS}


# ---- one mechanism at a time --------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, window, rot, page, scaling, softcap, loop", [
    (3, 1, 12, 20, 40, 6, 16, (4.0, 1.0, 4.0, 48), 3.0, None),      # sizes that are multiples of nothing
    (2, 2, 16, 8, 17, 16, 8, None, None, None),                     # the whole head rotated, no cap
    (4, 2, 32, 32, 65, 16, 16, (8.0, 1.0, 4.0, 64), None, None),    # no cap, keys and values of one size
    (6, 2, 128, 64, 64, 64, 16, (8.0, 1.0, 4.0, 64), 6.0, None),    # the tensor-core form, a window of a key tile
    (4, 1, 64, 128, 129, 0, 32, None, 5.0, None),                   # no rotation
    (2, 1, 128, 128, 200, 128, 16, None, None, None),               # heads of 128 without a cap
    (1, 1, 8, 8, 1, 8, 16, None, None, None),                       # a token sees itself alone
    (2, 1, 16, 32, 33, 8, 16, None, 4.0, (0, 1, 2)),
])
def test_windowed_attention_alone(tmp_path, dtype, heads, kv_heads, dim, vdim, window, rot, page, scaling, softcap, loop):
    gm.window_case(tmp_path, dtype, "cuda", heads, kv_heads, dim, vdim, window, rot, page, scaling, softcap, n=260, loop=loop)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, rot, page, scaling", [
    (4, 2, 16, 12, 8, 16, (4.0, 64, 8.0, 1.0)),
    (3, 3, 12, 20, 12, 8, (2.0, 32, 4.0, 0.5)),
    (8, 2, 64, 32, 32, 16, (8.0, 64, 32.0, 1.0)),       # the tensor-core form
    (2, 1, 128, 128, 64, 16, None),                     # heads of 128
    (2, 1, 16, 16, 0, 16, None),
])
def test_attention_with_biases_alone(tmp_path, dtype, heads, kv_heads, dim, vdim, rot, page, scaling):
    gm.left_case(tmp_path, dtype, "cuda", heads, kv_heads, dim, vdim, rot, page, scaling, n=260)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, dim, vdim, tau, rank", [
    (2, 16, 32, 16.0, 4),           # the chunked form in bfloat16
    (1, 64, 128, 4.0, 16),
    (2, 48, 80, 1.0, 7),
    (3, 10, 7, 1.0, 1),             # sizes the chunked form does not take
    (1, 12, 12, 4.0, 9),
])
def test_gated_linear_attention_alone(tmp_path, dtype, heads, dim, vdim, tau, rank):
    gm.gated_linear_case(tmp_path, dtype, "cuda", heads, dim, vdim, tau, rank, n=260)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, dim, vdim, kv_rank, q_rank, page", [
    (3, 16, 20, 24, 12, 16), (1, 12, 12, 20, 30, 8), (6, 32, 48, 96, 64, 16), (2, 64, 16, 512, 600, 32)])
def test_latent_attention_alone(tmp_path, dtype, heads, dim, vdim, kv_rank, q_rank, page):
    gm.latent_case(tmp_path, dtype, "cuda", heads, dim, vdim, kv_rank, q_rank, page, n=260)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts, top, ff", [(12, 3, 20), (5, 1, 24), (4, 4, 8), (1, 1, 16), (64, 6, 32)])
def test_experts_alone(tmp_path, dtype, experts, top, ff):
    gm.experts_case(tmp_path, dtype, "cuda", experts, top, ff)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("loop", [None, (0, 4, 1), (1, 3, 2), (2, 2, 5), (3, 4, 3)])
def test_the_loop_alone(tmp_path, dtype, loop):
    gm.loop_case(tmp_path, dtype, "cuda", loop)


# ---- the new kernels against their equations ----------------------------------------------------------

class _Step:
    """What the recurrence's kernels read of a step: sequences of ``lens`` tokens (one-token sequences first)."""

    def __init__(self, lens, slots):
        cu = [0]
        for n in lens:
            cu.append(cu[-1] + n)
        dev = dict(dtype=torch.int32, device="cuda")
        self.cu_q_lens, self.state_slots = torch.tensor(cu, **dev), torch.tensor(slots, **dev)
        self.num_seqs, self.num_decode = len(lens), sum(n == 1 for n in lens)


def plain_gla(x, z, heads, d, e, tau, weight, eps):
    """The mixer between its projections: x [n, 2 H (D + E)] rows [q | k | v | g], z [n, H D]; also the state left."""
    n = x.shape[0]
    q, k = (x[:, i * heads * d:(i + 1) * heads * d].reshape(n, heads, d) for i in range(2))
    v = x[:, 2 * heads * d:2 * heads * d + heads * e].reshape(n, heads, e)
    alpha = torch.exp(torch.nn.functional.logsigmoid(z) / tau).reshape(n, heads, d)
    o = pg.rms_norm(pg.gated_linear_recurrence(q * d ** -0.5, k, v, alpha), weight, eps).reshape(n, heads * e)
    s = torch.zeros(heads, d, e, dtype=x.dtype)
    for t in range(n):
        s = alpha[t][:, :, None] * s + k[t][:, :, None] * v[t][:, None, :]
    return o * pg.silu(x[:, 2 * heads * d + heads * e:2 * heads * (d + e)]), s


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, d, e, rank, tau, spread", [
    (3, 16, 16, 4, 16.0, 1.0), (2, 128, 256, 16, 16.0, 3.0), (4, 64, 80, 8, 4.0, 2.0), (1, 256, 192, 24, 16.0, 1.0),
    (2, 48, 144, 1, 1.0, 1.0), (5, 7, 11, 3, 2.0, 1.0), (2, 20, 300, 5, 16.0, 1.0), (1, 300, 8, 6, 8.0, 1.0),
    (2, 64, 64, 8, 1.0, 6.0),        # decays from one to e^-20 and below, side by side and from token to token
])
def test_the_gated_linear_attention_kernels_alone(heads, d, e, rank, tau, spread, dtype):
    """Sequences of unequal lengths in one launch (decoded tokens beside portions, lengths at and beside a
    chunk's 64 and a run's 16), then their next tokens from the state the launch left."""
    from deterministic_inference_b200.kernels import ops
    dt = getattr(torch, dtype)
    g = torch.Generator().manual_seed(heads * 31 + d + e)
    rounds = [[1, 1, 64, 65, 2, 200, 16], [1, 64, 1, 63, 129, 3, 17], [1, 1, 1, 1, 1, 1, 33]]
    order = [[0, 1, 2, 3, 4, 5, 6], [3, 0, 4, 2, 1, 5, 6], [5, 4, 3, 2, 1, 0, 6]]       # which sequence brings which count
    for lens, who in zip(rounds, order):                                                 # one-token sequences come first
        pairs = sorted(zip(lens, who), key=lambda p: p[0] != 1)
        lens[:], who[:] = [p[0] for p in pairs], [p[1] for p in pairs]
    total = [sum(l[w.index(i)] for l, w in zip(rounds, order)) for i in range(7)]
    width = 2 * heads * (d + e)
    seqs = [(torch.randn(n, width, generator=g) * 0.8).to(dt) for n in total]
    hidden = [torch.randn(n, rank, generator=g) for n in total]
    a2 = (torch.randn(rank, heads * d, generator=g) * spread / math.sqrt(rank)).to(dt)
    bias = torch.randn(heads * d, generator=g) * spread + 1.0
    weight = 1.0 + 0.3 * torch.randn(e, generator=g)
    want = [plain_gla(s.double(), h.double() @ a2.double() + bias.double(), heads, d, e, tau, weight.double(), 1e-5)
            for s, h in zip(seqs, hidden)]
    state = torch.zeros(8, heads * d * e, device="cuda")
    state[0] = float("nan")               # slot 0 is no request's: nothing reads it
    done = [0] * 7
    got = [[] for _ in range(7)]
    for lens, who in zip(rounds, order):
        rows = torch.cat([seqs[i][done[i]:done[i] + n] for n, i in zip(lens, who)]).cuda().contiguous()
        hid = torch.cat([hidden[i][done[i]:done[i] + n] for n, i in zip(lens, who)]).cuda().contiguous()
        out = ops.gated_linear_attention(rows, hid, 0, a2.cuda(), bias.cuda(), tau, weight.cuda(), state,
                                         _Step(lens, [i + 1 for i in who]), heads, d, e, 1e-5, dt)
        at = 0
        for n, i in zip(lens, who):
            got[i].append(out[at:at + n].double().cpu())
            done[i] += n
            at += n
    for i, (ref, left) in enumerate(want):
        err = (torch.cat(got[i]) - ref).abs()
        assert float(err.max()) <= (1e-4 if dtype == "float32" else 2e-2) * float(ref.abs().max()), (i, float(err.max()))
        # the state itself is float32 in both engines: it differs from the plain recurrence over the same rows
        # by far less than one bfloat16 rounding (below the least decay of the chunked form by no more than that)
        have = state[i + 1].double().cpu().view(heads, d, e)
        assert float((have - left).abs().max()) <= (5e-5 if spread < 4 else 6e-4) * float(left.abs().max()), i


def test_few_rows_read_the_projection_s_split_sums():
    """The decay map's input as columns behind the others, everything as partial sums of a split product: the
    bits of a stored matrix of the same sums."""
    from deterministic_inference_b200.kernels import ops
    heads, d, e, rank = 2, 32, 48, 5
    g = torch.Generator().manual_seed(5)
    width = 2 * heads * (d + e)
    parts = torch.randn(3, 50, width + 8, generator=g).cuda()
    total = (parts[0] + parts[1]) + parts[2]
    a2, bias, weight = torch.randn(rank, heads * d, generator=g).bfloat16().cuda(), torch.zeros(heads * d, device="cuda"), \
        torch.ones(e, device="cuda")
    outs = []
    for proj in (ops.SplitSum(parts, torch.float32), total):
        state = torch.zeros(4, heads * d * e, device="cuda")
        outs.append((ops.gated_linear_attention(proj, proj, width, a2, bias, 4.0, weight, state, _Step([1, 49], [2, 3]), heads,
                                                d, e, 1e-5, torch.bfloat16), state))
    assert torch.equal(outs[0][0], outs[1][0]) and torch.equal(outs[0][1], outs[1][1])


def test_a_padding_sequence_starts_from_zero_and_stores_nothing():
    from deterministic_inference_b200.kernels import ops
    heads, d, e = 2, 32, 32
    g = torch.Generator().manual_seed(3)
    x = torch.randn(70, 2 * heads * (d + e), generator=g).bfloat16().cuda()
    hid, a2 = torch.randn(70, 4, generator=g).cuda(), torch.randn(4, heads * d, generator=g).bfloat16().cuda()
    for lens in ([1], [70], [1, 69]):
        state = torch.full((2, heads * d * e), float("nan"), device="cuda")
        n = sum(lens)
        out = ops.gated_linear_attention(x[:n].contiguous(), hid[:n].contiguous(), 0, a2, torch.zeros(heads * d, device="cuda"),
                                         4.0, torch.ones(e, device="cuda"), state, _Step(lens, [0] * len(lens)), heads, d, e,
                                         1e-5, torch.bfloat16)
        assert bool(torch.isfinite(out.float()).all()) and bool(torch.isnan(state).all())


@pytest.mark.parametrize("rows, w", [(3, 72), (70, 100), (5, 1024), (9, 3000), (4, 4097), (2, 9001)])
def test_terms_biases_and_norms_of_the_stream(rows, w):
    """Every kind of term (a tensor of either type, split sums, with a bias, normed, both) and every norm."""
    from deterministic_inference_b200.kernels import ops
    g = torch.Generator().manual_seed(w)
    r = lambda *s: torch.randn(*s, generator=g)
    weights = [1.0 + 0.2 * r(w) for _ in range(4)]
    bias, parts, b16, f32, start = r(w), r(5, rows, w), r(rows, w).bfloat16(), r(rows, w), r(rows, w) + 0.7
    split = ops.SplitSum(parts.cuda(), torch.float32)
    cases = [
        (None, torch.zeros(rows, w).double()),
        (ops.BiasedTerm(b16.cuda(), bias.cuda()), b16.double() + bias.double()),
        (ops.NormedTerm(ops.BiasedTerm(split, bias.cuda()), weights[0].cuda(), 1e-5),
         pg.rms_norm(parts.double().sum(0) + bias.double(), weights[0].double(), 1e-5)),
        (ops.WeightedSum([(0.5, ops.NormedTerm(ops.BiasedTerm(split, bias.cuda()), weights[0].cuda(), 1e-5)),
                          (0.25, ops.NormedTerm(b16.cuda(), weights[1].cuda(), 1e-3)), (1.0, f32.cuda())]),
         0.5 * pg.rms_norm(parts.double().sum(0) + bias.double(), weights[0].double(), 1e-5)
         + 0.25 * pg.rms_norm(b16.double(), weights[1].double(), 1e-3) + f32.double()),
    ]
    for term, added in cases:
        want = start.double() + added
        normed = {None: want, "rms": pg.rms_norm(want, weights[3].double(), 1e-6),
                  "layer": pg.layer_norm(want, weights[3].double(), 1e-6)}
        for norm, ref in normed.items():
            for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 5e-3)):
                stream, out = start.clone().cuda(), torch.empty(rows, w, dtype=dt, device="cuda")
                ops.stream_terms_(stream, term, norm, weights[3].cuda(), 1e-6, out)
                torch.testing.assert_close(stream.double().cpu(), want, atol=1e-5, rtol=1e-5)
                torch.testing.assert_close(out.double().cpu(), ref, atol=tol, rtol=tol)
        if term is not None:
            torch.testing.assert_close(term.tensor().double().cpu(), added, atol=1e-5, rtol=1e-5)
            torch.testing.assert_close(ops.as_tensor(ops.gather_rows(term, torch.tensor([rows - 1, 0], dtype=torch.int32).cuda())
                                                     ).double().cpu(), added[[rows - 1, 0]], atol=1e-5, rtol=1e-5)


@pytest.mark.parametrize("t, experts, top", [(3, 8, 2), (70, 64, 6), (17, 1, 1), (5, 300, 32), (9, 5, 5)])
def test_the_router_weights_the_chosen_logits_alone(t, experts, top):
    from deterministic_inference_b200.kernels import ops
    logits = 4.0 * torch.randn(t, experts + 3, generator=torch.Generator().manual_seed(experts))
    ids, weights = ops.route_experts(logits.cuda(), None, experts, top, 1, 1, 1.0, 0.0, score="chosen_softmax")
    best = torch.topk(logits[:, :experts].double(), top, dim=-1)
    assert torch.equal(ids.long().cpu(), best.indices)
    torch.testing.assert_close(weights.double().cpu(), torch.softmax(best.values, dim=-1), atol=1e-7, rtol=1e-5)


@pytest.mark.parametrize("t, w, f, experts, top", [(5, 64, 32, 4, 2), (300, 256, 128, 8, 2), (2100, 256, 256, 16, 1),
                                                   (4096, 256, 512, 12, 3), (40, 72, 20, 6, 3), (1500, 512, 128, 4, 1)])
def test_experts_without_a_gate_in_bfloat16(t, w, f, experts, top):
    """All tile sizes of the grouped products (16 and 64 rows on mma.sync, 128 on tcgen05, CUDA cores for odd
    sizes) against the plain experts, rounding what is stored."""
    from deterministic_inference_b200.kernels import ops
    g = torch.Generator().manual_seed(t + w)
    bf = lambda *s, a=1.0: (torch.randn(*s, generator=g) * a).bfloat16()
    x, wu, wd = bf(t, w), bf(experts, f, w, a=1.5 / math.sqrt(w)), bf(experts, w, f, a=1.0 / math.sqrt(f))
    ids = torch.rand(t, experts, generator=g).topk(top, dim=-1).indices
    share = torch.softmax(torch.randn(t, top, generator=g), dim=-1)
    got = ops.routed_experts(x.cuda(), ids.int().cuda(), share.cuda(), wu.cuda(), wd.cuda(), None, None, -1, torch.bfloat16,
                             gated=False).double().cpu()
    want = torch.zeros(t, w, dtype=torch.float64)
    for e in range(experts):
        weight = (share.double() * (ids == e)).sum(-1)
        rows = (ids == e).any(-1)
        h = pg.gelu(x[rows].double() @ wu[e].double().T).bfloat16().double()
        want[rows] += weight[rows, None] * (h @ wd[e].double().T)
    err = (got - want).abs().max()
    assert float(err) <= 1e-2 * float(want.abs().max()), float(err)
    ops.check_kernel_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("q_rank, rank, rot", [(36, 24, 8), (600, 520, 0), (16, 96, 32)])
def test_latent_rows_with_and_without_a_rotated_part(q_rank, rank, rot, dtype):
    from deterministic_inference_b200.kernels import ops
    dt = getattr(torch, dtype)
    g = torch.Generator().manual_seed(rank)
    t, page = 21, 8
    proj = torch.randn(t, q_rank + rank + rot + 5, generator=g).to(dt)
    wq, wc = 1.0 + 0.2 * torch.randn(q_rank, generator=g), 1.0 + 0.2 * torch.randn(rank, generator=g)
    pos = torch.arange(100, 100 + t, dtype=torch.int32)
    slots = torch.arange(page, page + t, dtype=torch.int32)
    slots[3] = -1
    freqs = pg.plain_frequencies(rot, 1000.0) if rot else None
    cache = torch.zeros(4, page * (rank + rot), dtype=dt, device="cuda")
    cq = ops.latent_rows(proj.cuda(), 0, q_rank, wq.cuda(), q_rank, rank, rot, wc.cuda(), 1e-5,
                         torch.tensor(freqs).cuda() if rot else None, pos.cuda(), cache, slots.cuda(), page, dt, amplitude=1.2)
    tol = 1e-4 if dtype == "float32" else 2e-2
    x = proj.double()
    torch.testing.assert_close(cq.double().cpu(), pg.rms_norm(x[:, :q_rank], wq.double(), 1e-5), atol=tol, rtol=tol)
    want = pg.rms_norm(x[:, q_rank:q_rank + rank], wc.double(), 1e-5)
    if rot:
        key = pg.rotate_halves(x[:, None, q_rank + rank:q_rank + rank + rot], pos, freqs, 1.2)[:, 0]
        want = torch.cat([want, key], dim=-1)
    want[3] = 0.0                           # no slot: nothing is stored
    have = cache.view(-1, rank + rot)[page:page + t].double().cpu()
    torch.testing.assert_close(have, want, atol=tol, rtol=tol)


def test_one_gate_number_per_head():
    from deterministic_inference_b200.kernels import ops
    g = torch.Generator().manual_seed(8)
    for dt in (torch.float32, torch.bfloat16):
        x, gate = torch.randn(9, 3 * 20, generator=g).to(dt), torch.randn(2, 9, 11, generator=g)
        got = ops.sigmoid_gate_(x.clone().cuda(), ops.SplitSum(gate.cuda(), dt), 4, 20)
        want = x.double().view(9, 3, 20) * torch.sigmoid(gate.sum(0)[:, 4:7].to(dt).double())[:, :, None]
        torch.testing.assert_close(got.double().cpu(), want.view(9, 60), atol=1e-5, rtol=5e-3)


# ---- whole models ------------------------------------------------------------------------------------------

CASES = {       # configuration -> request lengths, seed
    "k1": ([1, 2, 17, 64, 131, 200], 31),
    "k2": ([5, 33, 65, 150], 32),
    "k3": ([3, 22, 63, 130, 260], 33),
    "k4": ([2, 30, 75, 150], 36),
}


@pytest.fixture(scope="module")
def plain_logits(model_dirs):
    out = {}
    for name, (lens, seed) in CASES.items():
        cfg, w = pg.read_model_dir(model_dirs[name])
        reqs = gu.requests(cfg["vocab"], lens, seed)
        out[name] = (cfg, w, reqs, [pg.forward(cfg, w, r) for r in reqs])
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CASES))
def test_whole_models_under_all_cuttings(name, dtype, model_dirs):
    cfg, _ = pg.read_model_dir(model_dirs[name])
    lens, seed = CASES[name]
    gm.compare(model_dirs[name], gu.requests(cfg["vocab"], lens, seed), dtype, "cuda", gu.CONFIGS[name]["page_size"],
               tail=110, what=name, cuda_graphs=False)


def check_rows(got, exact):
    for (key, pos), row in got.items():
        e = exact[int(key.lstrip("xyz")[1:])]
        err = float(gm.row_errors(row, e[pos]))
        assert err <= 1e-4 * float(e.std()), f"request {key} position {pos}: {err:.4g}, logits {float(e.std()):.3g}"


@pytest.mark.parametrize("name", ["k1", "k3"])
def test_replay_all_cuttings(name, model_dirs, plain_logits, tmp_path):
    cfg, w, reqs, exact = plain_logits[name]
    trace = ru.Trace()
    ru.mixed(trace, reqs)                             # sizes the pool; four live requests at most
    ru.whole(trace, reqs)
    ru.last_one_by_one(trace, reqs, tail=150)         # long decoding
    ru.portions(trace, reqs)
    out = ru.run_trace(model_dirs[name], "float32", trace, tmp_path / "out", page_size=gu.CONFIGS[name]["page_size"])
    got = ru.read_rows(out, trace, cfg["vocab"])
    for kind in "mwtp":
        for i, r in enumerate(reqs):
            assert all((f"{kind}{i}", p) in got for p in range(len(r))), (kind, i)
    check_rows(got, exact)


def all_experts(name, out_dir):
    """The configuration with every expert chosen: a bfloat16 router may decide a close call the other way, and
    every later token then differs (a float32 engine routes as configured)."""
    config = copy.deepcopy(gu.CONFIGS[name]["config"])
    for layer in config["layers"]:
        if layer.get("mlp") is not None:
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return gu.write_model(config, gu.CONFIGS[name]["seed"], out_dir)


@pytest.mark.parametrize("dtype", DTYPES)
def test_replay_with_captured_graphs(dtype, model_dirs, tmp_path):
    """The step function as generation runs it: pure-decode steps replayed as captured CUDA graphs."""
    name = "k3"
    d = model_dirs[name] if dtype == "float32" else all_experts(name, tmp_path / "all")
    cfg, w = pg.read_model_dir(d)
    same = gu.requests(cfg["vocab"], [100] * 4, 41)
    other = gu.requests(cfg["vocab"], [33, 120, 77], 42)
    reqs = same + other
    exact = [pg.forward(cfg, w, r) for r in reqs]
    trace = ru.Trace()
    for prefix in ("", "x"):
        ru.lockstep(trace, same, portion=48, tail=30, prefix=prefix)
    ru.mixed(trace, reqs)
    out = ru.run_trace(d, dtype, trace, tmp_path / "out", page_size=gu.CONFIGS[name]["page_size"], cuda_graphs=True)
    got = ru.read_rows(out, trace, cfg["vocab"])
    if dtype == "float32":
        check_rows(got, exact)
        return
    bounds = [max(3.0 * float(gm.row_errors(pg.forward(cfg, w, r, rnd=pg.as_stored_bf16), e).max()), 2e-2 * float(e.std()))
              for r, e in zip(reqs, exact)]
    for (key, pos), row in got.items():
        i = int(key.lstrip("xyz")[1:])
        err = float(gm.row_errors(row, exact[i][pos]))
        assert err <= bounds[i], f"request {key} position {pos}: {err:.4g} exceeds {bounds[i]:.4g}"


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_stream_after_every_layer_run(dtype, model_dirs):
    """The residual stream stays float32 whatever the engine's type; a layer that runs three times counts three
    times."""
    d = model_dirs["k3"]
    cfg, w = pg.read_model_dir(d)
    (toks,) = gu.requests(cfg["vocab"], [90], 5)
    runner = gu.runner_for(d, dtype, "cuda", 8, [90], cuda_graphs=False)
    seen = []

    def hook(entry, hidden, residual):
        term = hidden.tensor() if hasattr(hidden, "tensor") else hidden
        assert residual.dtype == torch.float32
        seen.append((residual + term.float()).double().cpu())
    runner.model.after_layer = hook
    routes = {}
    gu.replay(runner, [toks], [[(0, 90)]], routes)
    choose = gm.following([routes[0][k] for k in sorted(routes[0])]) if dtype == "bfloat16" else None
    want = []
    pg.forward(cfg, w, toks, rnd=pg.as_stored_bf16 if dtype == "bfloat16" else (lambda x: x), layers_out=want, choose=choose)
    assert len(seen) == len(want) == 9
    for i, (got, ref) in enumerate(zip(seen, want)):
        err, scale = float((got - ref).abs().max()), float(ref.abs().max())
        assert err <= (1e-4 if dtype == "float32" else 6e-2) * scale, f"layer run {i}: {err:.4g} of {scale:.4g}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CASES))
def test_greedy_generation_through_the_entry_point(name, dtype, model_dirs, tmp_path):
    from deterministic_inference_b200 import Engine, EngineConfig, SamplingParams
    d = model_dirs[name] if dtype == "float32" else all_experts(name, tmp_path / "all")
    cfg, w = pg.read_model_dir(d)
    prompts = gu.requests(cfg["vocab"], [3, 40, 9, 77, 15], 9)
    new = 30
    eng = Engine(EngineConfig(model_path=str(d), dtype=dtype, kv_pool_tokens=384, page_size=gu.CONFIGS[name]["page_size"],
                              max_reqs=3, max_seq_len=160, max_prefill_tokens=48))
    outs = eng.generate(prompts, SamplingParams(max_new_tokens=new, ignore_eos=True))
    eng.cache.check_invariants()
    for p, o in zip(prompts, outs):
        assert len(o.token_ids) == new
        # one plain pass over the engine's own continuation: every token is the best one given what
        # stands before it, or so close to it that rounding can flip the choice
        logits = pg.forward(cfg, w, p + o.token_ids)[len(p) - 1:-1]
        spread = float(logits.std())
        for k, t in enumerate(o.token_ids):
            gap = float(logits[k].max() - logits[k, t])
            assert gap <= (1e-3 if dtype == "float32" else 0.2) * spread, f"token {k} of {len(p)}+: {gap:.3g} below the best"
