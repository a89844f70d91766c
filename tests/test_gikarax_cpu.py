"""The Gikarax design without a GPU: configuration and registry, weights, the cache manager's share (a cache
per pass of the loop), and the engine's host logic with the kernel wrappers replaced by plain PyTorch
restatements (fixture ``torch_ops``), against the plain implementation of ``tests/plain_gikarax.py``."""

import copy

import pytest
import torch

from deterministic_inference_b200.config import EngineConfig, SamplingParams
from deterministic_inference_b200.config.gikarax_config import GikaraxConfig
from deterministic_inference_b200.config.model_config import ConfigError
from deterministic_inference_b200.engine import Engine, SequenceInput
from deterministic_inference_b200.models.registry import build_model, config_from_dir
from deterministic_inference_b200.parts.position import RotaryEmbedding
from deterministic_inference_b200.parts.registry import BuildContext
from deterministic_inference_b200.parts.spec import CompositeSpec, PagedKVSpec, ScheduleEntry, StateSpec
from deterministic_inference_b200.weights.loader import WeightsError, load_weights
from tests import gikarax_mechanisms as gm
from tests import gikarax_util as gu
from tests import plain_gikarax as pg


@pytest.fixture(scope="module")
def model_dirs(tmp_path_factory):
    return {name: gu.write_tiny(name, tmp_path_factory.mktemp(f"gikarax_{name}")) for name in gu.CONFIGS}


# ---- configuration, registry, weights ---------------------------------------------------------

def test_the_registry_picks_the_design_by_its_name_and_reads_every_size(model_dirs):
    cfg = config_from_dir(model_dirs["k1"])
    assert isinstance(cfg, GikaraxConfig)
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.loop) == (150, 72, 2e-5, (1, 3, 2))
    plan = cfg.plan()
    assert [l.mixer.kind for l in plan.layers] == ["parallel", "masked_attention", "latent_attention", "masked_attention"]
    assert [l.feed_forward.kind for l in plan.layers] == ["routed_experts", "none", "routed_experts", "routed_experts"]
    assert {l.block.kind for l in plan.layers} == {"parallel_f32_stream"}
    assert {l.mixer_norm.kind for l in plan.layers} | {plan.final_norm.kind} == {"stream_layer_norm"}
    # every run of a layer has a cache of its own; the loop's first layer takes the entry in each pass
    assert [(e.layer, e.cache, e.enters) for e in plan.schedule] == \
        [(0, 0, False), (1, 1, True), (2, 2, False), (1, 3, True), (2, 4, False), (3, 5, False)]
    left, right = (b.params for b in plan.layers[0].mixer.params["branches"])
    assert (left["num_heads"], left["num_kv_heads"], left["head_dim"], left["v_head_dim"], left["bias"], left["out_bias"]) == \
        (6, 3, 20, 12, True, True)
    assert left["position_encoding"].params["yarn"] == {"factor": 3.0, "original": 40, "fast": 6.0, "slow": 0.7}
    assert (right["num_heads"], right["head_dim"], right["v_head_dim"], right["tau"], right["decay_rank"]) == (3, 12, 20, 3.0, 5)
    assert plan.layers[0].mixer.params["scales"] == [0.5, 0.5]
    a = plan.layers[1].mixer.params
    assert (a["mask"], a["mask_size"], a["softcap"], a["gate"], a["sink_score"], a["qk_norm_eps"]) == \
        ("window", 21, 4.0, "head", 0.0, 2e-5)
    assert a["position_encoding"].params["scaling"] == {"factor": 4.0, "low": 1.0, "high": 5.0, "original": 32}
    m = plan.layers[2].mixer.params
    assert (m["num_heads"], m["head_dim"], m["rot_dim"], m["v_head_dim"], m["kv_rank"], m["q_rank"], m["gate"]) == \
        (3, 20, 0, 12, 28, 36, True)
    f = plan.layers[3].feed_forward.params
    assert (f["num_experts"], f["top"], f["intermediate_size"], f["activation"], f["score"], f["correction"]) == \
        (9, 4, 12, "gelu", "chosen_softmax", False)
    assert GikaraxConfig.from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()
    assert config_from_dir(model_dirs["k4"]).plan().layers[1].mixer.params["position_encoding"] is None
    for name in gu.CONFIGS:
        c = config_from_dir(model_dirs[name])
        specs = build_model(c, torch.float32, "cpu").tensor_specs()
        assert sum(torch.Size(s.shape).numel() for s in specs) == c.num_parameters()


def test_the_rank_of_the_decay_map_comes_from_the_checkpoint(model_dirs, tmp_path):
    import json
    import shutil
    shutil.copytree(model_dirs["k3"], tmp_path / "m")
    raw = json.loads((tmp_path / "m" / "config.json").read_text())
    for layer in raw["layers"]:
        if layer["type"] == "parallel":
            layer["mixer"]["right"].pop("decay_rank")
    (tmp_path / "m" / "config.json").write_text(json.dumps(raw))
    cfg = config_from_dir(tmp_path / "m")
    assert [layer["mixer"]["right"]["decay_rank"] for layer in cfg.layers if layer["type"] == "parallel"] == [16, 8]
    with pytest.raises(ConfigError, match="rank of the decay map"):
        GikaraxConfig.from_dict(raw)


@pytest.mark.parametrize("change, why", [
    (lambda c: c.pop("width"), "width"),
    (lambda c: c["norm"].pop("eps"), "norm.eps"),
    (lambda c: c["layers"][0].update(type="delta"), "type 'delta'"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "mixer.right"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("slow"), "scaling lacks"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(tau=0.0), "tau"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=14), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(high=0.5), "high > low"),
    (lambda c: c["layers"][2]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][2]["mlp"].update(kind="dense"), "kind 'dense'"),
    (lambda c: c["layers"][2]["mlp"]["router"].update(top=6), "more than 5 experts"),
    (lambda c: c["loop"].update(stop=5), "does not fit"),
    (lambda c: c["loop"].update(times=0), "does not fit"),
])
def test_a_configuration_that_does_not_fit_is_refused_with_the_reason(change, why):
    raw = copy.deepcopy(gu.CONFIGS["k1"]["config"])
    change(raw)
    with pytest.raises(ConfigError, match=why):
        GikaraxConfig.from_dict(raw)


def test_missing_misshapen_and_unexpected_tensors_are_listed(model_dirs, tmp_path):
    from safetensors.torch import load_file, save_file
    d = model_dirs["k1"]
    model = build_model(config_from_dir(d), torch.float32, "cpu")
    stored = load_file(str(d / "model.safetensors"))

    def refused(change, why):
        t = dict(stored)
        change(t)
        save_file(t, str(tmp_path / "model.safetensors"))
        with pytest.raises(WeightsError, match=why):
            load_weights(tmp_path, model.tensor_specs(), model.plan, torch.float32, "cpu")

    refused(lambda t: t.pop("loop.in"), "missing tensors")
    refused(lambda t: t.pop("l0.mix.left.o.b"), "missing tensors")
    refused(lambda t: t.update({"l1.norm2": stored["l1.norm1"].clone()}), "unexpected tensors")
    refused(lambda t: t.update({"l1.mix.g": stored["l1.mix.q"].clone()}), "wrong shapes")
    refused(lambda t: t.update({"l2.mlp.e0.gate": stored["l2.mlp.e0.up"].clone()}), "unexpected tensors")


def test_a_plan_whose_entries_replace_the_stream_needs_the_part_that_does():
    cfg = GikaraxConfig.from_dict(gu.CONFIGS["k4"]["config"])
    plan = cfg.plan()
    assert plan.stream_entry is None and "loop.in" in plan.ignored_names
    import dataclasses
    bad = dataclasses.replace(plan, schedule=(ScheduleEntry(layer=0, cache=0, enters=True),))
    with pytest.raises(ValueError, match="no stream entry"):
        bad.validate()


@pytest.mark.parametrize("dims, base, scaling", [
    (16, 10000.0, (4.0, 1.0, 4.0, 64)), (64, 500000.0, (8.0, 1.0, 4.0, 8192)), (12, 777.0, (3.0, 0.5, 6.0, 24)),
    (8, 100.0, (1.0, 1.0, 2.0, 16)), (24, 777.0, None)])
def test_stretched_frequencies(dims, base, scaling):
    sc = None if scaling is None else dict(zip(gu.STRETCHED, scaling))
    rope = RotaryEmbedding(BuildContext(torch.float32, torch.device("cpu")), head_dim=dims, rotary_dim=dims, theta=base,
                           scaling=sc)
    assert rope.frequency_list() == pytest.approx(pg.stretched_frequencies(dims, base, sc), rel=1e-13)
    assert rope.amplitude == 1.0


# ---- caches ---------------------------------------------------------------------------------------

def test_every_pass_of_the_loop_has_pages_and_states_of_its_own(model_dirs):
    model = build_model(config_from_dir(model_dirs["k3"]), torch.bfloat16, "cpu")
    specs = model.cache_specs()
    assert sorted(specs) == list(range(9))             # one layer in front, three passes over two layers, two behind
    window = PagedKVSpec(2, 128, 40, v_head_dim=64)
    assert specs[0] == PagedKVSpec(1, 96, None, v_head_dim=0)
    pair = CompositeSpec((PagedKVSpec(2, 64, None, v_head_dim=80), StateSpec((2 * 64 * 128,))))
    assert [specs[i] for i in (1, 3, 5)] == [window] * 3 and [specs[i] for i in (2, 4, 6)] == [pair] * 3
    assert specs[8].members[1] == StateSpec((4 * 48 * 32,))
    assert model.state_on_device()


# ---- one mechanism at a time, through the engine's step function on the CPU ---------------------------

@pytest.mark.parametrize("heads, kv_heads, dim, vdim, window, rot, page, scaling, softcap, loop", [
    (3, 1, 12, 20, 40, 6, 16, (4.0, 1.0, 4.0, 48), 3.0, None),
    (2, 2, 16, 8, 17, 16, 8, None, None, None),                  # the whole head rotated, no cap
    (2, 1, 12, 12, 32, 0, 16, None, 5.0, None),                  # no rotation, a window of two pages
    (1, 1, 8, 8, 1, 8, 16, None, None, None),                    # a token sees itself alone
    (2, 1, 16, 12, 33, 8, 16, None, 4.0, (0, 1, 2)),
])
def test_windowed_attention_alone(tmp_path, torch_ops, heads, kv_heads, dim, vdim, window, rot, page, scaling, softcap, loop):
    gm.window_case(tmp_path, "float32", "cpu", heads, kv_heads, dim, vdim, window, rot, page, scaling, softcap, n=130, loop=loop)


@pytest.mark.parametrize("heads, kv_heads, dim, vdim, rot, page, scaling", [
    (4, 2, 16, 12, 8, 16, (4.0, 64, 8.0, 1.0)), (3, 3, 12, 20, 12, 8, (2.0, 32, 4.0, 0.5)), (2, 1, 16, 16, 0, 16, None)])
def test_attention_with_biases_alone(tmp_path, torch_ops, heads, kv_heads, dim, vdim, rot, page, scaling):
    gm.left_case(tmp_path, "float32", "cpu", heads, kv_heads, dim, vdim, rot, page, scaling, n=120)


@pytest.mark.parametrize("heads, dim, vdim, tau, rank", [(2, 16, 24, 16.0, 4), (3, 10, 7, 1.0, 1), (1, 12, 12, 4.0, 9)])
def test_gated_linear_attention_alone(tmp_path, torch_ops, heads, dim, vdim, tau, rank):
    gm.gated_linear_case(tmp_path, "float32", "cpu", heads, dim, vdim, tau, rank, n=140)


@pytest.mark.parametrize("heads, dim, vdim, kv_rank, q_rank, page", [(3, 16, 20, 24, 12, 16), (1, 12, 12, 20, 30, 8)])
def test_latent_attention_alone(tmp_path, torch_ops, heads, dim, vdim, kv_rank, q_rank, page):
    gm.latent_case(tmp_path, "float32", "cpu", heads, dim, vdim, kv_rank, q_rank, page, n=130)


@pytest.mark.parametrize("experts, top, ff", [(12, 3, 20), (5, 1, 24), (4, 4, 8), (1, 1, 16)])
def test_experts_alone(tmp_path, torch_ops, experts, top, ff):
    gm.experts_case(tmp_path, "float32", "cpu", experts, top, ff)


@pytest.mark.parametrize("loop", [None, (0, 4, 1), (1, 3, 2), (0, 2, 3), (2, 2, 5), (3, 4, 2)])
def test_the_loop_alone(tmp_path, torch_ops, loop):
    gm.loop_case(tmp_path, "float32", "cpu", loop)


# ---- whole models: the engine's host logic on the CPU -------------------------------------------------

@pytest.mark.parametrize("name", list(gu.CONFIGS))
def test_cuttings_batches_and_reused_slots_on_cpu(name, model_dirs, torch_ops):
    cfg, _ = pg.read_model_dir(model_dirs[name])
    reqs = gu.requests(cfg["vocab"], [60, 37, 2, 26, 45], 3)
    gm.compare(model_dirs[name], reqs, "float32", "cpu", gu.CONFIGS[name]["page_size"], tail=35, what=name)


def test_the_stream_after_every_layer_run(model_dirs, torch_ops):
    """The float32 residual stream (pending terms added) after each run of a layer."""
    from tests.torch_kernels import _plain
    cfg, w = pg.read_model_dir(model_dirs["k3"], torch.float32)
    (toks,) = gu.requests(cfg["vocab"], [19], 5)
    want = []
    pg.forward(cfg, w, toks, layers_out=want)
    runner = gu.runner_for(model_dirs["k3"], "float32", "cpu", 8, [19])
    seen = []
    runner.model.after_layer = lambda e, hidden, residual: seen.append(residual + _plain(hidden))
    s = runner.cache.allocate_slot()
    runner.step([SequenceInput(s, toks, 0, [18])])
    assert len(seen) == len(want) == 9
    for i, (got, ref) in enumerate(zip(seen, want)):
        assert got.dtype == torch.float32
        torch.testing.assert_close(got, ref, atol=3e-4, rtol=1e-4, msg=lambda m, i=i: f"layer run {i}: {m}")


def generate_plain(cfg, w, prompt, new):
    ids = list(prompt)
    for _ in range(new):
        ids.append(int(torch.argmax(pg.forward(cfg, w, ids)[-1])))
    return ids[len(prompt):]


@pytest.mark.parametrize("name", ["k1", "k4"])
def test_greedy_generation_through_the_entry_point_on_cpu(name, model_dirs, torch_ops):
    d = model_dirs[name]
    cfg, w = pg.read_model_dir(d, torch.float32)
    prompts = gu.requests(cfg["vocab"], [3, 20, 9], 7)
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
    cfg = preset("gikarax_tiny")
    assert isinstance(cfg, GikaraxConfig)
    out = tmp_path / "model"
    assert main(["random", "--preset", "gikarax_tiny", "--seed", "3", "--out", str(out)]) == 0
    back = config_from_dir(out)
    assert back.to_dict() == cfg.to_dict()
    model = build_model(back, torch.float32, "cpu")
    load_weights(out, model.tensor_specs(), model.plan, torch.float32, "cpu")
