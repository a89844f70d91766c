"""Typed configuration of the Nedupel design, read from the keys of its config.json.

A pre-norm decoder with a scaled token embedding and a residual stream in float32 that takes every
sublayer's output times one constant (x <- x + m mixer(norm1(x)), then x <- x + m ff(norm2(x)), RMS
norms with weights stored around zero) and two kinds of mixer in any order: "latent_attention", causal
softmax attention whose keys and values are rebuilt from a small latent per token, with a rotated key
part shared by the heads (interleaved pairs, frequencies blended by pair index), where a layer may
read the cached rows of an earlier one; and "retention", a matrix state per head that shrinks by
one constant a token and is read without a softmax, behind it a per-head norm and a silu gate.  The feed-forward is dense with a squared relu, or a mixture of
experts with limited gates whose choice is a table of the token ids.  The head has a matrix of its
own; the logits are scaled by a constant.

config.json keys: ``architecture``, ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``,
``residual_mult``, ``logit_scale`` and ``layers``: per layer ``type``, ``mixer`` (latent_attention:
``heads``, ``dim``, ``rot_dim``, ``vdim``, ``kv_rank``, ``scale``, ``rot.base``, ``rot.dims``,
``rot.scaling`` (``factor``, ``original``, ``fast``, ``slow``; optional) and optionally ``kv_from``: the
index of the earlier layer whose cached rows this layer reads; retention: ``heads``, ``dim``, ``vdim``,
``decay``, ``rot.base``, ``rot.dims``) and ``mlp`` (``kind`` "dense" with ``ff``, or "moe" with
``expert.ff``, ``expert.limit``, ``router.experts``, ``router.top``; or null).  ``max_positions`` is
optional (no part of the design needs a longest position; it bounds the engine's block tables).
Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*`` (an integer
table ``l<i>.mlp.table`` [vocab, top] among them), ``final.norm``, ``head``.
"""

from __future__ import annotations

import copy
import json
from dataclasses import dataclass
from pathlib import Path

from ..parts.spec import LayerSpec, ModelPlan, PartSpec, ScheduleEntry
from .model_config import ConfigError

# fixed by the design
SWISH_ALPHA = 1.702              # an expert's gate is g * sigmoid(1.702 g)
NORM_WEIGHT_OFFSET = 1.0         # norm weights are stored around zero
DEFAULT_MAX_POSITIONS = 1 << 20


def _positive(what: str, v) -> int:
    if not isinstance(v, int) or isinstance(v, bool) or v < 1:
        raise ConfigError(f"{what} must be a positive integer, got {v!r}")
    return v


def _check_rot(what: str, rot, size: int) -> None:
    if not isinstance(rot, dict) or "base" not in rot or "dims" not in rot:
        raise ConfigError(f"{what}: rot.base and rot.dims are needed")
    dims = rot["dims"]
    if not isinstance(dims, int) or isinstance(dims, bool) or dims < 0 or dims % 2 or dims > size:
        raise ConfigError(f"{what}: rot.dims {dims!r} must be even and at most {size}")
    if float(rot["base"]) <= 0:
        raise ConfigError(f"{what}: rot.base must be positive")


def _check_latent(i: int, m: dict, layers: list) -> None:
    what = f"layer {i}"
    for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"):
        _positive(f"{what}: mixer.{k}", m.get(k))
    if "scale" not in m:
        raise ConfigError(f"{what}: mixer.scale is missing")
    _check_rot(what, m.get("rot"), m["rot_dim"])
    if m["rot"]["dims"] != m["rot_dim"]:
        raise ConfigError(f"{what}: rot.dims {m['rot']['dims']} differs from rot_dim {m['rot_dim']}")
    sc = m["rot"].get("scaling")
    if sc is not None:
        missing = [k for k in ("factor", "original", "fast", "slow") if k not in sc]
        if missing:
            raise ConfigError(f"{what}: rot.scaling lacks {missing}")
        if min(float(sc[k]) for k in ("factor", "original", "fast", "slow")) <= 0 or float(m["rot"]["base"]) == 1.0:
            raise ConfigError(f"{what}: rot.scaling needs positive numbers and a base other than 1")
    j = m.get("kv_from")
    if j is None:
        return
    if not isinstance(j, int) or isinstance(j, bool) or not 0 <= j < i:
        raise ConfigError(f"{what}: kv_from {j!r} names no earlier layer")
    other = layers[j].get("mixer") or {}
    if layers[j].get("type") != "latent_attention" or other.get("kv_from") is not None:
        raise ConfigError(f"{what}: kv_from {j} is not a latent attention with a latent of its own")
    for k in ("kv_rank", "rot_dim", "rot"):
        if other.get(k) != m.get(k):
            raise ConfigError(f"{what}: mixer.{k} differs from that of layer {j}, whose cached rows it reads")


def _check_retention(i: int, m: dict) -> None:
    for k in ("heads", "dim", "vdim"):
        _positive(f"layer {i}: mixer.{k}", m.get(k))
    _check_rot(f"layer {i}", m.get("rot"), m["dim"])
    if m["rot"].get("scaling") is not None:
        raise ConfigError(f"layer {i}: the rotation of a retention mixer has no scaling")
    decay = m.get("decay")
    if not isinstance(decay, list) or len(decay) != m["heads"]:
        raise ConfigError(f"layer {i}: mixer.decay must list {m['heads']} numbers")
    if not all(0.0 <= float(d) <= 1.0 for d in decay):
        raise ConfigError(f"layer {i}: mixer.decay {decay!r} must lie in [0, 1]")


def _check_mlp(i: int, mlp: dict) -> None:
    kind = mlp.get("kind")
    if kind == "dense":
        _positive(f"layer {i}: mlp.ff", mlp.get("ff"))
        return
    if kind != "moe":
        raise ConfigError(f"layer {i}: mlp.kind {kind!r} is not known ('dense', 'moe')")
    e, r = mlp.get("expert") or {}, mlp.get("router") or {}
    _positive(f"layer {i}: mlp.expert.ff", e.get("ff"))
    if "limit" not in e or not float(e["limit"]) > 0:
        raise ConfigError(f"layer {i}: mlp.expert.limit must be a positive number")
    for k in ("experts", "top"):
        _positive(f"layer {i}: mlp.router.{k}", r.get(k))
    if r["top"] > r["experts"]:
        raise ConfigError(f"layer {i}: router.top {r['top']} is more than {r['experts']} experts")


@dataclass(frozen=True)
class NedupelConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple                  # the ``layers`` list of config.json
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    logit_scale: float = 1.0
    max_positions: int = DEFAULT_MAX_POSITIONS
    architecture: str = "Nedupel"

    # ---- construction -----------------------------------------------------

    @classmethod
    def from_dict(cls, cfg: dict) -> "NedupelConfig":
        missing = [k for k in ("vocab", "width", "norm", "embedding", "residual_mult", "logit_scale", "layers")
                   if k not in cfg]
        if missing:
            raise ConfigError(f"config.json lacks required keys: {missing}")
        if not isinstance(cfg["norm"], dict) or "eps" not in cfg["norm"]:
            raise ConfigError("config.json: norm.eps is missing")
        if not isinstance(cfg["embedding"], dict) or "scale" not in cfg["embedding"]:
            raise ConfigError("config.json: embedding.scale is missing")
        layers = copy.deepcopy(list(cfg["layers"]))
        if not layers:
            raise ConfigError("config.json lists no layers")
        for i, layer in enumerate(layers):
            kind, mixer = layer.get("type"), layer.get("mixer") or {}
            if kind == "latent_attention":
                _check_latent(i, mixer, layers)
            elif kind == "retention":
                _check_retention(i, mixer)
            else:
                raise ConfigError(f"layer {i}: type {kind!r} is not known ('latent_attention', 'retention')")
            if layer.get("mlp") is not None:
                _check_mlp(i, layer["mlp"])
        out = cls(vocab=_positive("vocab", cfg["vocab"]), width=_positive("width", cfg["width"]),
                  norm_eps=float(cfg["norm"]["eps"]), layers=tuple(layers),
                  embedding_scale=float(cfg["embedding"]["scale"]), residual_mult=float(cfg["residual_mult"]),
                  logit_scale=float(cfg["logit_scale"]),
                  max_positions=_positive("max_positions", cfg.get("max_positions", DEFAULT_MAX_POSITIONS)),
                  architecture=str(cfg.get("architecture", "Nedupel")))
        if out.norm_eps <= 0:
            raise ConfigError("norm.eps must be positive")
        return out

    @classmethod
    def from_json(cls, model_dir) -> "NedupelConfig":
        return cls.from_dict(json.loads((Path(model_dir) / "config.json").read_text()))

    def to_dict(self) -> dict:
        """The config.json content that ``from_dict`` reads back unchanged."""
        out = {"architecture": self.architecture, "embedding": {"scale": self.embedding_scale},
               "layers": copy.deepcopy(list(self.layers)), "logit_scale": self.logit_scale,
               "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult, "vocab": self.vocab,
               "width": self.width}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        return out

    def validate(self) -> None:
        NedupelConfig.from_dict(self.to_dict())

    # ---- derived -----------------------------------------------------------

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    def num_parameters(self) -> int:
        w = self.width
        n = 2 * self.vocab * w + w
        for layer in self.layers:
            m, mlp = layer["mixer"], layer.get("mlp")
            n += w
            if layer["type"] == "latent_attention":
                n += m["heads"] * (m["dim"] + m["rot_dim"] + m["vdim"]) * w \
                    + m["heads"] * (m["dim"] + m["vdim"]) * m["kv_rank"]
                if m.get("kv_from") is None:
                    n += (m["kv_rank"] + m["rot_dim"]) * w + m["kv_rank"]
            else:
                n += m["heads"] * (2 * m["dim"] + 3 * m["vdim"]) * w
            if mlp is not None:
                n += w
                n += 2 * mlp["ff"] * w if mlp["kind"] == "dense" \
                    else mlp["router"]["experts"] * 3 * mlp["expert"]["ff"] * w
        return n

    # ---- the plan ------------------------------------------------------------

    def _mixer_spec(self, i: int) -> PartSpec:
        layer = self.layers[i]
        m, rot = layer["mixer"], layer["mixer"]["rot"]
        common = dict(prefix=f"l{i}.mix.", hidden_size=self.width, num_heads=m["heads"], head_dim=m["dim"],
                      v_head_dim=m["vdim"], norm_eps=self.norm_eps)
        if layer["type"] == "latent_attention":
            return PartSpec("latent_attention", dict(
                common, rot_dim=m["rot_dim"], kv_rank=m["kv_rank"], scale=float(m["scale"]),
                position_encoding=PartSpec("rope", dict(head_dim=m["rot_dim"], rotary_dim=rot["dims"],
                                                        theta=float(rot["base"]), yarn=rot.get("scaling"))),
                mask="causal", rotary_layout="pairs", own_latent=m.get("kv_from") is None))
        return PartSpec("retention", dict(
            common, decay=list(m["decay"]),
            position_encoding=None if not rot["dims"] else PartSpec("rope", dict(
                head_dim=m["dim"], rotary_dim=rot["dims"], theta=float(rot["base"])))))

    def _feed_forward_spec(self, i: int, mlp: dict) -> PartSpec:
        common = dict(prefix=f"l{i}.mlp.", hidden_size=self.width)
        if mlp["kind"] == "dense":
            return PartSpec("dense_mlp", dict(common, intermediate_size=mlp["ff"], activation="squared_relu"))
        r, e = mlp["router"], mlp["expert"]
        return PartSpec("routed_experts", dict(
            common, intermediate_size=e["ff"], num_experts=r["experts"], top=r["top"], route_scale=1.0,
            score="table", vocab_size=self.vocab, activation="limited_swish", limit=float(e["limit"]),
            alpha=SWISH_ALPHA))

    def plan(self) -> ModelPlan:
        w = self.width
        norm = dict(size=w, eps=self.norm_eps, weight_offset=NORM_WEIGHT_OFFSET)
        layers, ignored, schedule = [], [], []
        for i, layer in enumerate(self.layers):
            p, mlp = f"l{i}.", layer.get("mlp")
            if mlp is None:
                ff, ff_norm = PartSpec("none", {}), PartSpec("none", {})
                ignored.append(p + "norm2")
            else:
                ff = self._feed_forward_spec(i, mlp)
                ff_norm = PartSpec("stream_rms_norm", dict(name=p + "norm2", **norm))
            layers.append(LayerSpec(
                block=PartSpec("pre_norm_f32_stream", dict(branch_scale=self.residual_mult)),
                mixer=self._mixer_spec(i), feed_forward=ff,
                mixer_norm=PartSpec("stream_rms_norm", dict(name=p + "norm1", **norm)), feed_forward_norm=ff_norm))
            # a layer that reads another's latents runs on that layer's cache and writes nothing
            j = layer["mixer"].get("kv_from")
            schedule.append(ScheduleEntry(layer=i, cache=i if j is None else j, writes_cache=j is None))
        return ModelPlan(
            hidden_size=w, vocab_size=self.vocab,
            embedding=PartSpec("scaled_token_embedding", dict(name="embed", vocab_size=self.vocab, hidden_size=w,
                                                              scale=self.embedding_scale)),
            head=PartSpec("linear_head", dict(name="head", vocab_size=self.vocab, hidden_size=w,
                                              scale=self.logit_scale)),
            final_norm=PartSpec("stream_rms_norm", dict(name="final.norm", **norm)),
            layers=tuple(layers), schedule=tuple(schedule), max_positions=self.max_positions, eos_token_ids=(),
            ignored_names=tuple(ignored))
