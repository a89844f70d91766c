"""Tiny Gikarax models for the tests: configurations that differ in every size and option (also in values
that may happen to be equal or 1 elsewhere: one head or several, as many key heads as query heads or one,
key and value sizes equal or not, a full, a partial or no rotation, changed frequencies or plain ones, a
window of one token, a soft cap or none, one chosen expert or all of them, a layer without a feed-forward, a
loop over all layers, over some, of one pass, over none, or no loop), written with random weights by the
package's writer and then rescaled so that every mechanism weighs in the logits: streams of unit size,
scores that reach the soft cap, decays that neither forget everything nor nothing, routers whose choice
changes from token to token.  The schedules and the replay through the step function are those of
``tests/kipezen_util.py`` (they know no design)."""

from __future__ import annotations

import math
from pathlib import Path

from tests.kipezen_util import (last_one_by_one, mixed, portions, replay, requests, runner_for,  # noqa: F401
                                schedules, whole)

STRETCHED, BLENDED = ("factor", "low", "high", "original"), ("factor", "original", "fast", "slow")


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def rotation(base, dims, scaling, keys):
    rot = {"base": base, "dims": dims}
    if scaling is not None:
        rot["scaling"] = dict(zip(keys, scaling))
    return rot


def attention(heads, kv_heads, dim, vdim, window, rot, scaling=None, softcap=None, scale=None, mlp=None):
    """``rot``: (base, dims)."""
    return {"type": "attention", "mlp": mlp, "mixer": {
        "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
        "rot": rotation(*rot, scaling, STRETCHED), "scale": 3.0 / math.sqrt(dim) if scale is None else scale,
        "softcap": softcap}}


def left(heads, kv_heads, dim, vdim, rot, scaling=None, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rotation(*rot, scaling, BLENDED),
            "scale": 1.0 / math.sqrt(dim) if scale is None else scale}


def right(heads, dim, vdim, tau, rank):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "decay_rank": rank}


def parallel(left_half, right_half, mlp=None):
    return {"type": "parallel", "mixer": {"left": left_half, "right": right_half}, "mlp": mlp}


def latent(heads, dim, vdim, kv_rank, q_rank, scale=None, mlp=None):
    return {"type": "latent_attention", "mlp": mlp, "mixer": {
        "heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
        "scale": 1.0 / math.sqrt(dim) if scale is None else scale}}


def model(layers, vocab, width, eps=1e-5, loop=None):
    return {"architecture": "Gikarax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers,
            "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop))}


CONFIGS = {
    # sizes that are multiples of nothing (the kernels that take any size), partial rotations, a layer
    # without a feed-forward, a loop over the middle
    "k1": dict(page_size=16, seed=81, config=model([
        parallel(left(6, 3, 20, 12, (777.0, 10), scaling=(3.0, 40, 6.0, 0.7)), right(3, 12, 20, 3.0, 5), mlp=moe(6, 3, 28)),
        attention(5, 1, 12, 20, 21, (3000.0, 6), scaling=(4.0, 1.0, 5.0, 32), softcap=4.0, mlp=None),
        latent(3, 20, 12, 28, 36, mlp=moe(5, 2, 20)),
        attention(2, 2, 20, 12, 33, (500.0, 20), softcap=2.5, mlp=moe(9, 4, 12))],
        150, 72, eps=2e-5, loop=(1, 3, 2))),
    # what can be 1 is 1: one head, one expert, one pass over all layers, a decay exponent of 1, a map of
    # rank 1, a window of one token; plain frequencies over the whole head, no soft cap; pages of 32
    "k2": dict(page_size=32, seed=82, config=model([
        attention(1, 1, 48, 48, 1, (30000.0, 48), mlp=moe(1, 1, 48)),
        parallel(left(1, 1, 48, 48, (10000.0, 48)), right(1, 32, 32, 1.0, 1), mlp=moe(3, 3, 40)),
        latent(1, 32, 32, 48, 16, scale=0.3, mlp=moe(4, 1, 24))], 300, 96, eps=1e-6, loop=(0, 3, 1))),
    # sizes the tensor-core kernels take; three passes over two layers; pages of 8
    "k3": dict(page_size=8, seed=83, config=model([
        latent(8, 32, 48, 96, 64, mlp=moe(16, 4, 64)),
        attention(6, 2, 128, 64, 40, (10000.0, 32), scaling=(8.0, 1.0, 4.0, 64), softcap=6.0, mlp=moe(8, 2, 96)),
        parallel(left(8, 2, 64, 80, (500.0, 64), scaling=(2.0, 32, 4.0, 0.5)), right(2, 64, 128, 16.0, 16), mlp=moe(12, 1, 64)),
        attention(4, 4, 32, 32, 19, (300.0, 16), softcap=30.0, mlp=None),
        parallel(left(3, 3, 16, 32, (10000.0, 8)), right(4, 48, 32, 6.0, 8), mlp=None)],
        211, 128, eps=3e-6, loop=(1, 3, 3))),
    # a width that is a multiple of 4 only, odd head sizes, no rotation, no loop
    "k4": dict(page_size=16, seed=84, config=model([
        parallel(left(5, 5, 12, 20, (3000.0, 0)), right(3, 9, 7, 8.0, 3), mlp=moe(6, 2, 36)),
        attention(5, 5, 12, 20, 64, (3000.0, 0), softcap=3.0, mlp=moe(4, 4, 20)),
        latent(5, 7, 9, 20, 11, mlp=None)], 131, 100)),
}


def sharpen(model_dir) -> None:
    from safetensors.torch import load_file, save_file

    path = Path(model_dir) / "model.safetensors"
    tensors = load_file(str(path))

    def unit(t, gain):      # a matrix drawn with std 0.02 -> std gain / sqrt(inputs)
        return t.float() * (gain / (0.02 * math.sqrt(t.shape[-1])))

    for name, t in list(tensors.items()):
        end = name.split(".", 1)[-1] if name.startswith("l") and name[1].isdigit() else name
        x = None
        if name == "embed":
            x = t.float() * 50.0
        elif name.endswith("a2.b"):
            x = t.float() * 50.0 + 2.0                       # most channels keep most of the state
        elif name.endswith(".b"):
            x = t.float() * 15.0                             # biases of size 0.3
        elif t.dim() == 2:
            gain = {"mix.left.q": 2.0, "mix.left.k": 2.0, "mix.uq": 2.0, "mix.uk": 2.0, "mlp.router": 2.0, "mix.g": 2.0,
                    "head": 1.5}.get(end, 1.2)
            x = unit(t, gain)
        if x is not None:
            tensors[name] = x.to(t.dtype)
    save_file(tensors, str(path), metadata={"format": "pt"})


def write_model(config: dict, seed: int, out_dir, edit=None) -> Path:
    """Random weights, rescaled as for the tiny models, then changed by ``edit(tensors)`` (float32 in,
    stored as bfloat16)."""
    from safetensors.torch import load_file, save_file

    from deterministic_inference_b200.config.gikarax_config import GikaraxConfig
    from deterministic_inference_b200.weights import write_random_model

    write_random_model(GikaraxConfig.from_dict(config), seed, out_dir)
    sharpen(out_dir)
    if edit is not None:
        path = Path(out_dir) / "model.safetensors"
        stored = load_file(str(path))
        tensors = {k: v.float() for k, v in stored.items()}
        edit(tensors)
        save_file({k: v.to(stored[k].dtype).contiguous() for k, v in tensors.items()}, str(path),
                  metadata={"format": "pt"})
    return Path(out_dir)


def write_tiny(name: str, out_dir) -> Path:
    spec = CONFIGS[name]
    return write_model(spec["config"], spec["seed"], out_dir)
