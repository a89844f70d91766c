"""The Nedupel design on the GPU against the plain implementation of ``tests/plain_nedupel.py``:
each mechanism alone (``tests/nedupel_mechanisms.py``), the new kernels alone against their equations,
then whole models under every cutting (whole prompts, the last tokens one by one, portions down to two
tokens, mixed batches in a pool so small that pages and slots are used again), in float32 through
``bin/trace_run`` and in bfloat16 through the step function; with captured graphs; and greedy
generation through ``Engine.generate``."""

import math

import pytest
import torch

from tests import nedupel_mechanisms as nm
from tests import nedupel_util as nu
from tests import plain_nedupel as pn
from tests import replay_util as ru

pytestmark = pytest.mark.gpu

DTYPES = ("float32", "bfloat16")


@pytest.fixture(scope="module")
def model_dirs(tmp_path_factory):
    return {name: nu.write_tiny(name, tmp_path_factory.mktemp(f"nedupel_{name}")) for name in nu.CONFIGS}


# ---- one mechanism at a time --------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, dim, rot_dim, vdim, rank, page, scaling, shared", [
    (3, 16, 8, 20, 24, 16, (4.0, 64, 8.0, 1.0), False),        # sizes that are multiples of nothing
    (2, 12, 12, 12, 20, 8, None, False),                       # plain frequencies
    (4, 32, 16, 48, 64, 16, (2.0, 32, 4.0, 0.5), True),        # the tensor-core form; a second layer reads the rows
    (8, 64, 32, 32, 96, 32, (8.0, 64, 32.0, 1.0), True),
])
def test_latent_attention_alone(tmp_path, dtype, heads, dim, rot_dim, vdim, rank, page, scaling, shared):
    nm.latent_case(tmp_path, dtype, "cuda", heads, dim, rot_dim, vdim, rank, page, scaling, shared)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim, vdim, decay, rot", [
    (16, 32, (0.99, 0.9995), 8),              # the chunked form in bfloat16, a partial rotation
    (64, 128, (0.995, 0.9990234375), 64),     # the whole head rotated
    (48, 80, (1.0,), 20),                     # a decay that forgets nothing
    (10, 14, (0.995, 0.999), 0),              # sizes the chunked form does not take; no rotation
    (12, 9, (0.999, 0.9), 12),                # columns one at a time
])
def test_retention_alone(tmp_path, dtype, dim, vdim, decay, rot):
    nm.retention_case(tmp_path, dtype, "cuda", dim, vdim, decay, rot)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts, top, ff, limit", [(12, 3, 20, 0.5), (5, 1, 24, 1.0), (4, 4, 8, 0.7), (1, 1, 16, 0.3),
                                                     (64, 6, 32, 0.6)])
def test_experts_of_a_table_alone(tmp_path, dtype, experts, top, ff, limit):
    nm.experts_case(tmp_path, dtype, "cuda", experts, top, ff, limit)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff", [50, 192])
def test_squared_relu_alone(tmp_path, dtype, ff):
    nm.dense_case(tmp_path, dtype, "cuda", ff)


# ---- the new kernels against their equations ----------------------------------------------------------

class _Step:
    """What the retention kernels read of a step: sequences of ``lens`` tokens (one-token sequences first)
    behind ``done`` tokens each."""

    def __init__(self, lens, done, slots):
        cu = [0]
        for n in lens:
            cu.append(cu[-1] + n)
        dev = dict(dtype=torch.int32, device="cuda")
        self.cu_q_lens, self.state_slots = torch.tensor(cu, **dev), torch.tensor(slots, **dev)
        self.positions = torch.tensor([d + k for n, d in zip(lens, done) for k in range(n)], **dev)
        self.num_seqs, self.num_decode = len(lens), sum(n == 1 for n in lens)


def plain_retention(x, heads, d, e, decay, freqs, eps):
    """The mixer between its projections: x [n, 2 H (D + E)] rows [q | k | v | g]."""
    n = x.shape[0]
    q, k = (x[:, i * heads * d:(i + 1) * heads * d].reshape(n, heads, d) for i in range(2))
    v = x[:, 2 * heads * d:2 * heads * d + heads * e].reshape(n, heads, e)
    pos = torch.arange(n)
    q, k = pn.rotate_halves(q, pos, freqs), pn.rotate_halves(k, pos, freqs) * d ** -0.5
    o = pn.unit_rms(pn.retention_recurrence(q, k, v, decay), eps).reshape(n, heads * e)
    return o * pn.silu(x[:, 2 * heads * d + heads * e:])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, d, e, rot", [(3, 16, 16, 16), (2, 128, 256, 64), (4, 64, 80, 10), (1, 256, 192, 256),
                                              (2, 48, 144, 0), (5, 7, 11, 4), (2, 20, 300, 20), (1, 300, 8, 6)])
def test_the_retention_kernels_alone(heads, d, e, rot, dtype):
    """Sequences of unequal lengths in one launch (decoded tokens beside portions, lengths at and beside
    a chunk's 64), then their next tokens from the state the launch left."""
    from deterministic_inference_b200.kernels import ops
    dt = getattr(torch, dtype)
    g = torch.Generator().manual_seed(heads * 31 + d + e)
    freqs = pn.plain_frequencies(rot, 10000.0) if rot else []
    decay = [1.0 - 0.5 ** (2 + 2 * i) for i in range(heads)]
    rounds = [[1, 1, 64, 65, 2, 200], [1, 64, 1, 63, 129, 3], [1, 1, 1, 1, 1, 1]]
    order = [[0, 1, 2, 3, 4, 5], [3, 0, 4, 2, 1, 5], [5, 4, 3, 2, 1, 0]]       # which sequence brings which count
    for lens, who in zip(rounds, order):                                        # one-token sequences come first
        pairs = sorted(zip(lens, who), key=lambda p: p[0] != 1)
        lens[:], who[:] = [p[0] for p in pairs], [p[1] for p in pairs]
    total = [sum(l[w.index(i)] for l, w in zip(rounds, order)) for i in range(6)]
    width = 2 * heads * (d + e)
    seqs = [(torch.randn(n, width, generator=g) * 0.8).to(dt) for n in total]
    want = [plain_retention(s.double(), heads, d, e, decay, freqs, 1e-5) for s in seqs]
    state = torch.zeros(7, heads * d * e, device="cuda")
    state[0] = float("nan")               # slot 0 is no request's: nothing reads it
    freq = torch.tensor(freqs, dtype=torch.float32, device="cuda") if rot else None
    done = [0] * 6
    dec = torch.tensor(decay, dtype=torch.float32, device="cuda")
    got = [[] for _ in range(6)]
    for lens, who in zip(rounds, order):
        rows = torch.cat([seqs[i][done[i]:done[i] + n] for n, i in zip(lens, who)]).cuda().contiguous()
        step = _Step(lens, [done[i] for i in who], [i + 1 for i in who])
        out = ops.retention(rows, dec, freq, state, step, heads, d, e, 1e-5, dt)
        at = 0
        for n, i in zip(lens, who):
            got[i].append(out[at:at + n].double().cpu())
            done[i] += n
            at += n
    # the outputs of a unit norm times a gate: absolute errors of the outputs' own scale
    for i, ref in enumerate(want):
        err = (torch.cat(got[i]) - ref).abs()
        assert float(err.max()) <= (1e-4 if dtype == "float32" else 2e-2) * float(ref.abs().max()), (i, float(err.max()))
    # the state itself is float32 in both engines: what a bfloat16 engine leaves differs from the plain
    # recurrence over the same rows by far less than one bfloat16 rounding
    x = seqs[5].double()
    k = x[:, heads * d:2 * heads * d].reshape(-1, heads, d)
    k = pn.rotate_halves(k, torch.arange(len(x)), freqs) * d ** -0.5
    v = x[:, 2 * heads * d:2 * heads * d + heads * e].reshape(-1, heads, e)
    left = torch.zeros(heads, d, e, dtype=torch.float64)
    for t in range(len(x)):
        left = torch.tensor(decay).double()[:, None, None] * left + k[t][:, :, None] * v[t][:, None, :]
    have = state[6].double().cpu().view(heads, d, e)
    assert float((have - left).abs().max()) <= 3e-5 * float(left.abs().max())


def test_a_padding_sequence_starts_from_zero_and_stores_nothing():
    from deterministic_inference_b200.kernels import ops
    heads, d, e = 2, 32, 32
    x = torch.randn(70, 2 * heads * (d + e), generator=torch.Generator().manual_seed(3)).bfloat16().cuda()
    dec = torch.tensor([0.9, 0.99], device="cuda")
    for lens in ([1], [70], [1, 69]):
        state = torch.full((2, heads * d * e), float("nan"), device="cuda")
        out = ops.retention(x[:sum(lens)].contiguous(), dec, None, state, _Step(lens, [0] * len(lens), [0] * len(lens)), heads, d,
                            e, 1e-5, torch.bfloat16)
        assert bool(torch.isfinite(out.float()).all()) and bool(torch.isnan(state).all())


@pytest.mark.parametrize("t, w, f, experts, top", [(5, 64, 32, 4, 2), (300, 256, 128, 8, 2), (2100, 256, 128, 16, 1),
                                                   (4096, 256, 256, 12, 3), (40, 72, 20, 6, 3)])
def test_limited_experts_of_a_table_in_bfloat16(t, w, f, experts, top):
    """All tile sizes of the grouped products (16 and 64 rows on mma.sync, 128 on tcgen05, CUDA cores for
    odd sizes) against the plain experts, rounding what is stored."""
    from deterministic_inference_b200.kernels import ops
    g = torch.Generator().manual_seed(t + w)
    bf = lambda *s, a=1.0: (torch.randn(*s, generator=g) * a).bfloat16()
    x, wgu, wd = bf(t, w), bf(experts, 2 * f, w, a=1.5 / math.sqrt(w)), bf(experts, w, f, a=1.0 / math.sqrt(f))
    table = torch.rand(50, experts, generator=g).topk(top, dim=-1).indices.int()
    ids = torch.randint(0, 50, (t,), generator=g).int()
    choice = ops.TableChoice(ids.cuda(), table.cuda(), 1.0 / top)
    got = ops.routed_experts(x.cuda(), choice, None, wgu.cuda(), wd.cuda(), None, None, -1, torch.bfloat16,
                             limited=(0.7, 1.702)).double().cpu()
    want = torch.zeros(t, w, dtype=torch.float64)
    xd = x.double()
    for e in range(experts):
        rows = (table[ids.long()] == e).any(-1)
        gu = xd[rows] @ wgu[e].double().T
        a, b = gu[:, :f].clamp(max=0.7), gu[:, f:].clamp(-0.7, 0.7)
        h = (a * torch.sigmoid(1.702 * a) * (b + 1.0)).bfloat16().double()
        want[rows] += h @ wd[e].double().T / top
    err = (got - want).abs().max()
    assert float(err) <= 1e-2 * float(want.abs().max()), float(err)


@pytest.mark.parametrize("m, n, k", [(3, 96, 64), (64, 256, 128), (65, 384, 192), (500, 520, 264), (2048, 1024, 256),
                                     (4000, 4096, 512), (130, 36, 100)])
def test_squared_relu_product_in_bfloat16(m, n, k):
    from deterministic_inference_b200.kernels import ops
    g = torch.Generator().manual_seed(m + n)
    x, w = torch.randn(m, k, generator=g).bfloat16(), (torch.randn(n, k, generator=g) / math.sqrt(k)).bfloat16()
    got = ops.squared_relu_linear(x.cuda(), w.cuda(), torch.bfloat16)
    want = torch.relu(x.double() @ w.double().T).square()
    assert got.dtype == torch.bfloat16
    torch.testing.assert_close(got.double().cpu(), want, atol=1e-4, rtol=6e-3)
    ops.check_kernel_status()


# ---- whole models ------------------------------------------------------------------------------------------

CASES = {       # configuration -> request lengths, seed
    "n1": ([1, 2, 17, 64, 131, 260], 31),
    "n2": ([5, 33, 65, 200], 32),
    "n3": ([3, 22, 63, 130, 333], 33),
    "n4": ([2, 30, 75, 180], 36),
}


@pytest.fixture(scope="module")
def plain_logits(model_dirs):
    out = {}
    for name, (lens, seed) in CASES.items():
        cfg, w = pn.read_model_dir(model_dirs[name])
        reqs = nu.requests(cfg["vocab"], lens, seed)
        out[name] = (cfg, w, reqs, [pn.forward(cfg, w, r) for r in reqs])
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CASES))
def test_whole_models_under_all_cuttings(name, dtype, model_dirs):
    cfg, _ = pn.read_model_dir(model_dirs[name])
    lens, seed = CASES[name]
    nm.compare(model_dirs[name], nu.requests(cfg["vocab"], lens, seed), dtype, "cuda", nu.CONFIGS[name]["page_size"],
               tail=110, what=name, cuda_graphs=False)


def check_rows(got, plain, dtype, name):
    cfg, w, reqs, exact = plain
    bounds = [nm.bound_of(cfg, w, r, e, dtype) for r, e in zip(reqs, exact)]
    for (key, pos), row in got.items():
        i = int(key.lstrip("xyz")[1:])
        err = float(nm.row_errors(row, exact[i][pos]))
        assert err <= bounds[i], f"{name}: request {key} position {pos}: {err:.4g} exceeds {bounds[i]:.4g}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["n1", "n3"])
def test_replay_all_cuttings(name, dtype, model_dirs, plain_logits, tmp_path):
    cfg, w, reqs, _ = plain_logits[name]
    trace = ru.Trace()
    ru.mixed(trace, reqs)                             # sizes the pool; four live requests at most
    ru.whole(trace, reqs)
    ru.last_one_by_one(trace, reqs, tail=150)         # long decoding
    ru.portions(trace, reqs)
    out = ru.run_trace(model_dirs[name], dtype, trace, tmp_path / "out", page_size=nu.CONFIGS[name]["page_size"])
    got = ru.read_rows(out, trace, cfg["vocab"])
    for kind in "mwtp":
        for i, r in enumerate(reqs):
            assert all((f"{kind}{i}", p) in got for p in range(len(r))), (kind, i)
    check_rows(got, plain_logits[name], dtype, name)


@pytest.mark.parametrize("dtype", DTYPES)
def test_replay_with_captured_graphs(dtype, model_dirs, tmp_path):
    """The step function as generation runs it: pure-decode steps replayed as captured CUDA graphs."""
    name = "n3"
    cfg, w = pn.read_model_dir(model_dirs[name])
    same = nu.requests(cfg["vocab"], [120] * 4, 41)
    other = nu.requests(cfg["vocab"], [33, 150, 77], 42)
    reqs = same + other
    exact = [pn.forward(cfg, w, r) for r in reqs]
    trace = ru.Trace()
    for prefix in ("", "x"):
        ru.lockstep(trace, same, portion=48, tail=30, prefix=prefix)
    ru.mixed(trace, reqs)
    out = ru.run_trace(model_dirs[name], dtype, trace, tmp_path / "out", page_size=nu.CONFIGS[name]["page_size"],
                       cuda_graphs=True)
    check_rows(ru.read_rows(out, trace, cfg["vocab"]), (cfg, w, reqs, exact), dtype, name)


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_stream_after_every_layer(dtype, model_dirs):
    """The residual stream stays float32 whatever the engine's type."""
    cfg, w = pn.read_model_dir(model_dirs["n3"])
    (toks,) = nu.requests(cfg["vocab"], [90], 5)
    runner = nu.runner_for(model_dirs["n3"], dtype, "cuda", 8, [90], cuda_graphs=False)
    seen = []

    def hook(entry, hidden, residual):
        term = hidden.tensor() if hasattr(hidden, "tensor") else hidden
        assert residual.dtype == torch.float32
        seen.append((residual + term.float()).double().cpu())
    runner.model.after_layer = hook
    nu.replay(runner, [toks], [[(0, 90)]])
    want = []
    pn.forward(cfg, w, toks, layers_out=want)
    assert len(seen) == len(want) == 6
    for i, (got, ref) in enumerate(zip(seen, want)):
        err, scale = float((got - ref).abs().max()), float(ref.abs().max())
        assert err <= (1e-4 if dtype == "float32" else 4e-2) * scale, f"layer {i}: {err:.4g} of {scale:.4g}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CASES))
def test_greedy_generation_through_the_entry_point(name, dtype, model_dirs):
    from deterministic_inference_b200 import Engine, EngineConfig, SamplingParams
    d = model_dirs[name]
    cfg, w = pn.read_model_dir(d)
    prompts = nu.requests(cfg["vocab"], [3, 40, 9, 77, 15], 9)
    new = 30
    eng = Engine(EngineConfig(model_path=str(d), dtype=dtype, kv_pool_tokens=384, page_size=nu.CONFIGS[name]["page_size"],
                              max_reqs=3, max_seq_len=160, max_prefill_tokens=48))
    outs = eng.generate(prompts, SamplingParams(max_new_tokens=new, ignore_eos=True))
    eng.cache.check_invariants()
    for p, o in zip(prompts, outs):
        assert len(o.token_ids) == new
        # one plain pass over the engine's own continuation: every token is the best one given what
        # stands before it, or so close to it that rounding can flip the choice
        logits = pn.forward(cfg, w, p + o.token_ids)[len(p) - 1:-1]
        spread = float(logits.std())
        for k, t in enumerate(o.token_ids):
            gap = float(logits[k].max() - logits[k, t])
            assert gap <= (1e-3 if dtype == "float32" else 0.2) * spread, f"token {k} of {len(p)}+: {gap:.3g} below the best"
