"""Tiny Nedupel models for the tests: configurations that differ in every size and option (also in
values that may happen to be equal or 1 elsewhere: one head or several, key and value sizes equal or
not, a full, a partial or no rotation, blended frequencies or plain ones, latents read by one or by
several later layers with other head counts, one chosen expert or all of them, factors of 1, a decay of
1, a layer without a feed-forward, models of one kind of mixer only), written with random weights by
the package's writer and then rescaled so that every mechanism weighs in the logits: streams of unit
size, scores of unit size, gates that reach their limit.  The schedules and the replay through the
step function are those of ``tests/kipezen_util.py`` (they know no design)."""

from __future__ import annotations

import math
from pathlib import Path

from tests.kipezen_util import (last_one_by_one, mixed, portions, replay, requests, runner_for,  # noqa: F401
                                schedules, whole)


def moe(experts, top, ff, limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def latent(heads, dim, rot_dim, vdim, rank, base, scaling=None, scale=None, kv_from=None, mlp=None):
    """``scaling``: (factor, original, fast, slow)."""
    rot = {"base": base, "dims": rot_dim}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "rot": rot,
         "scale": scale if scale is not None else 1.0 / math.sqrt(dim + rot_dim)}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def retention(dim, vdim, decay, base, dims, mlp=None):
    return {"type": "retention", "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay),
                                           "rot": {"base": base, "dims": dims}}, "mlp": mlp}


def model(layers, vocab, width, eps=1e-5, embed=1.0, mult=1.0, logit=1.0):
    return {"architecture": "Nedupel", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"scale": embed}, "residual_mult": mult, "logit_scale": logit, "layers": layers}


YARN = (4.0, 96, 8.0, 1.0)

CONFIGS = {
    # sizes that are multiples of nothing (the kernels that take any size); a partial rotation in the
    # retention; a layer without a feed-forward; one latent read twice, by other head counts
    "n1": dict(page_size=16, seed=71, config=model([
        retention(20, 12, (0.9, 0.995, 0.9995), 777.0, 10, mlp=moe(6, 3, 28, 0.8)),
        latent(3, 20, 12, 28, 36, 3000.0, scaling=YARN, mlp=dense(100)),
        latent(5, 12, 12, 20, 36, 3000.0, scaling=YARN, kv_from=1, mlp=None),
        latent(2, 28, 12, 12, 36, 3000.0, scaling=YARN, kv_from=1, scale=0.3, mlp=moe(5, 2, 20, 1.3))],
        150, 72, eps=2e-5, embed=1.7, mult=0.55, logit=0.7)),
    # everything that can be 1 is 1: one head, one expert, one chosen expert, factors of 1, a decay that
    # forgets nothing; plain frequencies; the whole head rotated; pages of 32
    "n2": dict(page_size=32, seed=72, config=model([
        latent(1, 48, 16, 48, 48, 30000.0, mlp=moe(1, 1, 48, 2.0)),
        retention(32, 32, (1.0,), 10000.0, 32, mlp=moe(3, 3, 40, 0.5))], 300, 96, eps=1e-6)),
    # sizes the tensor-core kernels take; latents of two layers, read across other layers; pages of 8
    "n3": dict(page_size=8, seed=73, config=model([
        latent(4, 64, 32, 32, 96, 10000.0, scaling=(8.0, 64, 32.0, 1.0), mlp=dense(256)),
        retention(64, 128, (0.95, 0.9990234375), 10000.0, 32, mlp=moe(16, 4, 64, 1.1)),
        latent(8, 32, 16, 48, 64, 500.0, scaling=(2.0, 32, 4.0, 0.5), mlp=moe(8, 2, 96, 0.7)),
        latent(2, 32, 32, 80, 96, 10000.0, scaling=(8.0, 64, 32.0, 1.0), kv_from=0, mlp=moe(4, 1, 64, 0.7)),
        latent(4, 48, 16, 32, 64, 500.0, scaling=(2.0, 32, 4.0, 0.5), kv_from=2, mlp=dense(64)),
        retention(16, 48, (0.8, 0.9, 0.97, 0.998), 300.0, 16, mlp=None)],
        211, 128, eps=3e-6, embed=0.8, mult=0.4, logit=0.3)),
    # a width that is a multiple of 4 only, odd head sizes, retention without a rotation, no latents at all
    "n4": dict(page_size=16, seed=74, config=model([
        retention(9, 7, (0.99, 0.5, 0.999), 3000.0, 0, mlp=dense(36)),
        retention(48, 176, (0.9921875, 0.96875), 3000.0, 6, mlp=moe(9, 4, 28, 3.0))],
        131, 100, embed=2.0, mult=0.8, logit=2.0)),
}


def sharpen(model_dir) -> None:
    from safetensors.torch import load_file, save_file

    path = Path(model_dir) / "model.safetensors"
    tensors = load_file(str(path))
    for name, t in list(tensors.items()):
        leaf = name.rsplit(".", 1)[-1]
        x = None
        if name == "embed":
            x = t.float() * 50.0
        elif leaf == "norm1" or leaf == "norm2" or name == "final.norm":
            x = t.float() * 10.0                              # weights around zero of size 0.2
        elif t.dim() == 2 and t.is_floating_point():          # drawn with std 0.02 -> gain / sqrt(inputs)
            gain = {"q": 2.0, "uk": 1.5, "k": 1.5, "gate": 1.5, "head": 1.5}.get(leaf, 1.2)
            x = t.float() * (gain / (0.02 * math.sqrt(t.shape[-1])))
        if x is not None:
            tensors[name] = x.to(t.dtype)
    save_file(tensors, str(path), metadata={"format": "pt"})


def write_model(config: dict, seed: int, out_dir, edit=None) -> Path:
    """Random weights, rescaled as for the tiny models, then changed by ``edit(tensors)`` (float32 in,
    stored as bfloat16; the integer tables as they are)."""
    from safetensors.torch import load_file, save_file

    from deterministic_inference_b200.config.nedupel_config import NedupelConfig
    from deterministic_inference_b200.weights import write_random_model

    write_random_model(NedupelConfig.from_dict(config), seed, out_dir)
    sharpen(out_dir)
    if edit is not None:
        path = Path(out_dir) / "model.safetensors"
        stored = load_file(str(path))
        tensors = {k: v.float() if v.is_floating_point() else v for k, v in stored.items()}
        edit(tensors)
        save_file({k: v.to(stored[k].dtype).contiguous() for k, v in tensors.items()}, str(path),
                  metadata={"format": "pt"})
    return Path(out_dir)


def write_tiny(name: str, out_dir) -> Path:
    spec = CONFIGS[name]
    return write_model(spec["config"], spec["seed"], out_dir)
