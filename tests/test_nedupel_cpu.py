"""The Nedupel design without a GPU: configuration and registry, weights (integer tables among them),
the cache manager's share (one latent row per token, read by later layers; state slots), and the engine's
host logic with the kernel wrappers replaced by plain PyTorch restatements (fixture ``torch_ops``),
against the plain implementation of ``tests/plain_nedupel.py``."""

import copy

import pytest
import torch

from deterministic_inference_b200.config import EngineConfig, SamplingParams
from deterministic_inference_b200.config.model_config import ConfigError
from deterministic_inference_b200.config.nedupel_config import NedupelConfig
from deterministic_inference_b200.engine import Engine, SequenceInput
from deterministic_inference_b200.models.registry import build_model, config_from_dir
from deterministic_inference_b200.parts.position import RotaryEmbedding
from deterministic_inference_b200.parts.registry import BuildContext
from deterministic_inference_b200.parts.spec import PagedKVSpec, StateSpec
from deterministic_inference_b200.weights.loader import WeightsError, load_weights
from tests import nedupel_mechanisms as nm
from tests import nedupel_util as nu
from tests import plain_nedupel as pn


@pytest.fixture(scope="module")
def model_dirs(tmp_path_factory):
    return {name: nu.write_tiny(name, tmp_path_factory.mktemp(f"nedupel_{name}")) for name in nu.CONFIGS}


# ---- configuration, registry, weights ---------------------------------------------------------

def test_the_registry_picks_the_design_by_its_name_and_reads_every_size(model_dirs):
    cfg = config_from_dir(model_dirs["n1"])
    assert isinstance(cfg, NedupelConfig)
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.embedding_scale, cfg.residual_mult, cfg.logit_scale) == \
        (150, 72, 2e-5, 1.7, 0.55, 0.7)
    plan = cfg.plan()
    assert [l.mixer.kind for l in plan.layers] == ["retention"] + ["latent_attention"] * 3
    # layers 2 and 3 run on layer 1's cache and write nothing
    assert [(e.layer, e.cache, e.writes_cache) for e in plan.schedule] == \
        [(0, 0, True), (1, 1, True), (2, 1, False), (3, 1, False)]
    assert [l.feed_forward.kind for l in plan.layers] == ["routed_experts", "dense_mlp", "none", "routed_experts"]
    assert [(l.block.kind, l.block.params["branch_scale"]) for l in plan.layers] == [("pre_norm_f32_stream", 0.55)] * 4
    r = plan.layers[0].mixer.params
    assert (r["num_heads"], r["head_dim"], r["v_head_dim"], r["decay"], r["norm_eps"]) == \
        (3, 20, 12, [0.9, 0.995, 0.9995], 2e-5)
    assert r["position_encoding"].params == {"head_dim": 20, "rotary_dim": 10, "theta": 777.0}
    a, b = plan.layers[1].mixer.params, plan.layers[3].mixer.params
    assert (a["num_heads"], a["head_dim"], a["rot_dim"], a["v_head_dim"], a["kv_rank"], a["own_latent"]) == \
        (3, 20, 12, 28, 36, True)
    assert (b["num_heads"], b["head_dim"], b["v_head_dim"], b["own_latent"], b["scale"]) == (2, 28, 12, False, 0.3)
    assert (a["mask"], a["rotary_layout"]) == ("causal", "pairs")
    assert a["position_encoding"].params["yarn"] == {"factor": 4.0, "original": 96, "fast": 8.0, "slow": 1.0}
    f = plan.layers[0].feed_forward.params
    assert (f["num_experts"], f["top"], f["intermediate_size"], f["limit"], f["alpha"], f["score"], f["vocab_size"]) == \
        (6, 3, 28, 0.8, 1.702, "table", 150)
    assert plan.layers[1].feed_forward.params["activation"] == "squared_relu"
    assert plan.layers[0].mixer_norm.params["weight_offset"] == 1.0
    assert NedupelConfig.from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()
    assert config_from_dir(model_dirs["n4"]).plan().layers[0].mixer.params["position_encoding"] is None
    specs = build_model(cfg, torch.float32, "cpu").tensor_specs()
    assert sum(torch.Size(s.shape).numel() for s in specs if s.role != "index") == cfg.num_parameters()


@pytest.mark.parametrize("change, why", [
    (lambda c: c.pop("residual_mult"), "residual_mult"),
    (lambda c: c["embedding"].pop("scale"), "embedding.scale"),
    (lambda c: c["layers"][0].update(type="delta"), "type 'delta'"),
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.9]), "decay"),
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.9, 1.5, 0.5]), r"\[0, 1\]"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=22), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10), "differs from rot_dim"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("fast"), "scaling lacks"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"].update(kv_from=2), "names no earlier layer"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=0), "latent of its own"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=2), "latent of its own"),
    (lambda c: c["layers"][2]["mixer"].update(kv_rank=40), "kv_rank differs"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(base=10.0), "rot differs"),
    (lambda c: c["layers"][1]["mlp"].update(ff=0), "mlp.ff"),
    (lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0.0), "limit"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "more than 6 experts"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "kind 'gated'"),
])
def test_a_configuration_that_does_not_fit_is_refused_with_the_reason(change, why):
    raw = copy.deepcopy(nu.CONFIGS["n1"]["config"])
    change(raw)
    with pytest.raises(ConfigError, match=why):
        NedupelConfig.from_dict(raw)


def test_missing_misshapen_and_unexpected_tensors_and_tables_are_listed(model_dirs, tmp_path):
    from safetensors.torch import load_file, save_file
    d = model_dirs["n1"]
    cfg = config_from_dir(d)
    model = build_model(cfg, torch.float32, "cpu")
    tensors = load_weights(d, model.tensor_specs(), model.plan, torch.float32, "cpu")
    assert tensors["l0.mlp.table"].dtype == torch.int32 and tuple(tensors["l0.mlp.table"].shape) == (150, 3)
    assert all(len(set(row)) == 3 for row in tensors["l0.mlp.table"].tolist())
    assert "l2.mix.dkv" not in tensors
    stored = load_file(str(d / "model.safetensors"))

    def refused(change, why):
        t = dict(stored)
        change(t)
        save_file(t, str(tmp_path / "model.safetensors"))
        with pytest.raises(WeightsError, match=why):
            load_weights(tmp_path, model.tensor_specs(), model.plan, torch.float32, "cpu")

    refused(lambda t: t.pop("l1.mix.dkv.norm"), "missing tensors")
    refused(lambda t: t.update({"l2.mix.dkv": stored["l1.mix.dkv"].clone()}), "unexpected tensors")
    refused(lambda t: t.update({"l0.mlp.table": stored["l0.mlp.table"].float()}), "expected an integer type")
    refused(lambda t: t.update({"l0.mlp.table": stored["l0.mlp.table"] + 1}), r"expected integers in \[0, 6\)")
    refused(lambda t: t.update({"l0.mix.q": stored["l0.mlp.table"].clone()}), "expected a floating type|wrong shapes")


@pytest.mark.parametrize("dims, base, scaling", [
    (16, 10000.0, (4.0, 96, 8.0, 1.0)), (64, 500000.0, (2.0, 512, 32.0, 1.0)), (12, 3000.0, (40.0, 4096, 32.0, 1.0)),
    (4, 10.0, (8.0, 16, 2.0, 1.5)),       # lo and hi meet: the smallest width of the blend
    (32, 100.0, (3.0, 100000, 16.0, 0.5)), (8, 50.0, (1.0, 64, 4.0, 1.0)), (24, 777.0, None)])
def test_blended_frequencies(dims, base, scaling):
    sc = None if scaling is None else dict(zip(("factor", "original", "fast", "slow"), scaling))
    rope = RotaryEmbedding(BuildContext(torch.float32, torch.device("cpu")), head_dim=dims, rotary_dim=dims, theta=base,
                           yarn=sc)
    freqs, size = pn.yarn_frequencies(dims, base, sc)
    assert rope.frequency_list() == pytest.approx(freqs, rel=1e-13)
    assert rope.amplitude == pytest.approx(size, rel=1e-13)
    assert rope.frequencies().dtype == torch.float32
    # the table form carries the same frequencies and the amplitude
    table = RotaryEmbedding(BuildContext(torch.float32, torch.device("cpu")), head_dim=dims, rotary_dim=dims, theta=base,
                            yarn=sc, max_positions=5).rotary_table()
    if scaling is not None:
        want = torch.tensor(freqs, dtype=torch.float64) * 4
        torch.testing.assert_close(table[4].double(), size * torch.cat([want.cos(), want.sin()]), atol=1e-5, rtol=1e-5)


# ---- caches ---------------------------------------------------------------------------------------

def test_latent_rows_are_kept_once_and_read_by_later_layers(model_dirs):
    model = build_model(config_from_dir(model_dirs["n3"]), torch.bfloat16, "cpu")
    specs = model.cache_specs()
    assert sorted(specs) == [0, 1, 2, 5]              # layers 3 and 4 own no cache
    assert specs[0] == PagedKVSpec(1, 96 + 32, None, v_head_dim=0)
    assert specs[2] == PagedKVSpec(1, 64 + 16, None, v_head_dim=0)
    assert specs[1] == StateSpec((2 * 64 * 128,)) and specs[5] == StateSpec((4 * 16 * 48,))
    assert model.state_on_device()
    # a reader whose rows would be of another size than the owner's is refused
    raw = copy.deepcopy(nu.CONFIGS["n3"]["config"])
    plan = NedupelConfig.from_dict(raw).plan()
    plan.layers[3].mixer.params.update(kv_rank=64)
    from deterministic_inference_b200.models.decoder import DecoderModel
    with pytest.raises(ValueError, match="another kind"):
        DecoderModel(plan, torch.float32, "cpu").cache_specs()


# ---- one mechanism at a time, through the engine's step function on the CPU ---------------------------

@pytest.mark.parametrize("heads, dim, rot_dim, vdim, rank, page, scaling, shared", [
    (3, 16, 8, 20, 24, 16, (4.0, 64, 8.0, 1.0), False),
    (2, 12, 12, 12, 20, 8, None, False),                       # plain frequencies
    (2, 16, 8, 16, 24, 16, (2.0, 32, 4.0, 0.5), True),         # a second layer reads the rows
])
def test_latent_attention_alone(tmp_path, torch_ops, heads, dim, rot_dim, vdim, rank, page, scaling, shared):
    nm.latent_case(tmp_path, "float32", "cpu", heads, dim, rot_dim, vdim, rank, page, scaling, shared, n=150)


@pytest.mark.parametrize("dim, vdim, decay, rot", [(16, 24, (0.99, 0.9995), 8), (12, 8, (1.0,), 12), (10, 14, (0.995, 0.999), 0)])
def test_retention_alone(tmp_path, torch_ops, dim, vdim, decay, rot):
    nm.retention_case(tmp_path, "float32", "cpu", dim, vdim, decay, rot, n=140)


@pytest.mark.parametrize("experts, top, ff, limit", [(12, 3, 20, 0.5), (5, 1, 24, 1.0), (4, 4, 8, 0.7), (1, 1, 16, 0.3)])
def test_experts_of_a_table_alone(tmp_path, torch_ops, experts, top, ff, limit):
    nm.experts_case(tmp_path, "float32", "cpu", experts, top, ff, limit)


def test_squared_relu_alone(tmp_path, torch_ops):
    nm.dense_case(tmp_path, "float32", "cpu", 50)


# ---- whole models: the engine's host logic on the CPU -------------------------------------------------

@pytest.mark.parametrize("name", list(nu.CONFIGS))
def test_cuttings_batches_and_reused_slots_on_cpu(name, model_dirs, torch_ops):
    cfg, _ = pn.read_model_dir(model_dirs[name])
    reqs = nu.requests(cfg["vocab"], [70, 41, 2, 26, 55], 3)
    nm.compare(model_dirs[name], reqs, "float32", "cpu", nu.CONFIGS[name]["page_size"], tail=45, what=name)


def test_the_stream_after_every_layer(model_dirs, torch_ops):
    """The float32 residual stream (pending term added) after each layer."""
    from tests.torch_kernels import _plain
    cfg, w = pn.read_model_dir(model_dirs["n3"], torch.float32)
    (toks,) = nu.requests(cfg["vocab"], [19], 5)
    want = []
    pn.forward(cfg, w, toks, layers_out=want)
    runner = nu.runner_for(model_dirs["n3"], "float32", "cpu", 8, [19])
    seen = []
    runner.model.after_layer = lambda e, hidden, residual: seen.append(residual + _plain(hidden))
    s = runner.cache.allocate_slot()
    runner.step([SequenceInput(s, toks, 0, [18])])
    assert len(seen) == len(want) == 6
    for i, (got, ref) in enumerate(zip(seen, want)):
        assert got.dtype == torch.float32
        torch.testing.assert_close(got, ref, atol=3e-4, rtol=1e-4, msg=lambda m, i=i: f"layer {i}: {m}")


def generate_plain(cfg, w, prompt, new):
    ids = list(prompt)
    for _ in range(new):
        ids.append(int(torch.argmax(pn.forward(cfg, w, ids)[-1])))
    return ids[len(prompt):]


@pytest.mark.parametrize("name", ["n1", "n4"])
def test_greedy_generation_through_the_entry_point_on_cpu(name, model_dirs, torch_ops):
    d = model_dirs[name]
    cfg, w = pn.read_model_dir(d, torch.float32)
    prompts = nu.requests(cfg["vocab"], [3, 20, 9], 7)
    want = [generate_plain(cfg, w, p, 10) for p in prompts]
    eng = Engine(EngineConfig(model_path=str(d), dtype="float32", device="cpu", kv_pool_tokens=96, page_size=16,
                              max_reqs=2, max_seq_len=64, max_prefill_tokens=12, cuda_graphs=False,
                              async_scheduling=False))
    outs = eng.generate(prompts, SamplingParams(max_new_tokens=10, ignore_eos=True))
    assert [o.token_ids for o in outs] == want
    eng.cache.check_invariants()


def test_the_command_line_writes_a_model_folder_the_registry_reads_back(tmp_path):
    from deterministic_inference_b200.__main__ import main
    from deterministic_inference_b200.config import preset
    cfg = preset("nedupel_tiny")
    assert isinstance(cfg, NedupelConfig)
    out = tmp_path / "model"
    assert main(["random", "--preset", "nedupel_tiny", "--seed", "3", "--out", str(out)]) == 0
    back = config_from_dir(out)
    assert back.to_dict() == cfg.to_dict()
    model = build_model(back, torch.float32, "cpu")
    load_weights(out, model.tensor_specs(), model.plan, torch.float32, "cpu")


def test_an_older_build_of_one_library_does_not_take_another_ones(tmp_path, monkeypatch):
    """Compiling a library removes ITS older builds; a library whose name starts with the same letters
    keeps its own."""
    from deterministic_inference_b200.kernels import build
    for name in ("libdib200_gemm_bf16_0123456789abcdef.so", "libdib200_gemm_bf16_large_0123456789abcdef.so"):
        (tmp_path / name).write_bytes(b"")
    monkeypatch.setattr(build, "_find_built", lambda name: None)
    monkeypatch.setattr(build, "library_path", lambda name: tmp_path / f"libdib200_{name}_ffff456789abcdef.so")

    class Done:
        returncode = 0

        def __init__(self, cmd, **_):
            from pathlib import Path
            Path(cmd[cmd.index("-o") + 1]).write_bytes(b"")

        def communicate(self):
            return "", None
    monkeypatch.setattr(build.subprocess, "Popen", Done)
    monkeypatch.setattr(build, "_nvcc", lambda: "nvcc")
    build.compile_library("gemm_bf16", verbose=False)
    assert sorted(p.name for p in tmp_path.glob("*.so")) == [
        "libdib200_gemm_bf16_ffff456789abcdef.so", "libdib200_gemm_bf16_large_0123456789abcdef.so"]
