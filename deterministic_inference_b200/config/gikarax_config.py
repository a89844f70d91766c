"""Typed configuration of the Gikarax design, read from the keys of its config.json.

A decoder with an unscaled token embedding and a residual stream in float32, whose layers have ONE layer
norm (a weight, no bias) that both sublayers read: x <- x + (mixer(h) + ff(h)), h = norm1(x).  Layers
``loop.start`` .. ``loop.stop`` - 1 run ``loop.times`` times in a row with the same weights and a cache of
their own for each pass; in front of every pass the stream becomes W_in [x; x0], x0 the embedding's
output.  Three kinds of mixer in any order: "attention" (sliding window, q and k normed per head, rotation
with stretched long wavelengths, capped scores, a sink of score 0, one gate number per head), "parallel"
(causal attention with biases and blended frequencies beside gated linear attention, each RMS-normed over
the width and halved) and "latent_attention" (causal, keys and values rebuilt from a small latent per
token, queries through a latent too, no positions, an element-wise output gate).  The feed-forward is a
mixture of experts without gates (erf gelu), weighted by the softmax over the chosen logits.  The head has
a matrix of its own.

config.json keys: ``architecture``, ``vocab``, ``width``, ``norm.eps``, ``loop`` (``start``, ``stop``,
``times``; or null) and ``layers``: per layer ``type``, ``mixer`` (attention: ``heads``, ``kv_heads``,
``dim``, ``vdim``, ``scale``, ``softcap``, ``mask.size``, ``rot.base``, ``rot.dims``, ``rot.scaling``
(``factor``, ``low``, ``high``, ``original``; optional); parallel: ``left`` (``heads``, ``kv_heads``, ``dim``,
``vdim``, ``scale``, ``rot`` with ``scaling`` of ``factor``, ``original``, ``fast``, ``slow``, optional) and
``right`` (``heads``, ``dim``, ``vdim``, ``tau``); latent_attention: ``heads``, ``dim``, ``vdim``,
``kv_rank``, ``q_rank``, ``scale``) and ``mlp`` (``kind`` "moe", ``expert.ff``, ``router.experts``,
``router.top``; or null).  The rank of the gated linear attention's decay map is the one size config.json
does not give: it is read from the checkpoint tensor's shape (``l<i>.mix.right.a1``), or from an optional
``right.decay_rank`` (configurations made in code).  ``max_positions`` is optional (no part of the design
needs a longest position; it bounds the engine's block tables).  Tensor names: ``embed``, ``loop.in``,
``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""

from __future__ import annotations

import copy
import json
from dataclasses import dataclass
from pathlib import Path
from typing import Optional

from ..parts.spec import LayerSpec, ModelPlan, PartSpec, ScheduleEntry
from .model_config import ConfigError

# fixed by the design
BRANCH_SCALE = 0.5               # the two normed branches of a parallel mixer are averaged
SINK_SCORE = 0.0                 # the score of the windowed attention's sink
DEFAULT_MAX_POSITIONS = 1 << 20

STRETCHED = ("factor", "low", "high", "original")     # keys of rot.scaling in "attention"
BLENDED = ("factor", "original", "fast", "slow")      # in the left half of "parallel"


def _positive(what: str, v) -> int:
    if not isinstance(v, int) or isinstance(v, bool) or v < 1:
        raise ConfigError(f"{what} must be a positive integer, got {v!r}")
    return v


def _positive_number(what: str, v) -> float:
    if not isinstance(v, (int, float)) or isinstance(v, bool) or not v > 0:
        raise ConfigError(f"{what} must be a positive number, got {v!r}")
    return float(v)


def _check_heads(what: str, m: dict) -> None:
    for k in ("heads", "kv_heads", "dim", "vdim"):
        _positive(f"{what}.{k}", m.get(k))
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"{what}.heads {m['heads']} is not a multiple of kv_heads {m['kv_heads']}")
    if "scale" not in m:
        raise ConfigError(f"{what}.scale is missing")


def _check_rot(what: str, m: dict, keys: tuple) -> None:
    rot = m.get("rot")
    if rot is None:
        return
    if not isinstance(rot, dict) or "base" not in rot or "dims" not in rot:
        raise ConfigError(f"{what}.rot.base and {what}.rot.dims are needed")
    dims = rot["dims"]
    if not isinstance(dims, int) or isinstance(dims, bool) or dims < 0 or dims % 2 or dims > m["dim"]:
        raise ConfigError(f"{what}.rot.dims {dims!r} must be even and at most {m['dim']}")
    _positive_number(f"{what}.rot.base", rot["base"])
    sc = rot.get("scaling")
    if sc is None:
        return
    missing = [k for k in keys if k not in sc]
    if missing:
        raise ConfigError(f"{what}.rot.scaling lacks {missing}")
    for k in keys:
        if k not in ("low", "high"):
            _positive_number(f"{what}.rot.scaling.{k}", sc[k])
    if "low" in keys and float(sc["high"]) <= float(sc["low"]):
        raise ConfigError(f"{what}.rot.scaling needs high > low")
    if "fast" in keys and float(rot["base"]) == 1.0:
        raise ConfigError(f"{what}.rot.base of blended frequencies is not 1")


def _check_layer(i: int, layer: dict) -> None:
    kind, m = layer.get("type"), layer.get("mixer") or {}
    if kind == "attention":
        _check_heads(f"layer {i}: mixer", m)
        _check_rot(f"layer {i}: mixer", m, STRETCHED)
        _positive(f"layer {i}: mixer.mask.size", (m.get("mask") or {}).get("size"))
        if m.get("softcap") is not None:
            _positive_number(f"layer {i}: mixer.softcap", m["softcap"])
    elif kind == "parallel":
        for k in ("left", "right"):
            if not isinstance(m.get(k), dict):
                raise ConfigError(f"layer {i}: mixer.{k} is missing")
        _check_heads(f"layer {i}: left", m["left"])
        _check_rot(f"layer {i}: left", m["left"], BLENDED)
        for k in ("heads", "dim", "vdim"):
            _positive(f"layer {i}: right.{k}", m["right"].get(k))
        _positive_number(f"layer {i}: right.tau", m["right"].get("tau"))
    elif kind == "latent_attention":
        for k in ("heads", "dim", "vdim", "kv_rank", "q_rank"):
            _positive(f"layer {i}: mixer.{k}", m.get(k))
        if "scale" not in m:
            raise ConfigError(f"layer {i}: mixer.scale is missing")
    else:
        raise ConfigError(f"layer {i}: type {kind!r} is not known ('attention', 'parallel', 'latent_attention')")
    mlp = layer.get("mlp")
    if mlp is None:
        return
    if mlp.get("kind") != "moe":
        raise ConfigError(f"layer {i}: mlp.kind {mlp.get('kind')!r} is not known (only 'moe')")
    _positive(f"layer {i}: mlp.expert.ff", (mlp.get("expert") or {}).get("ff"))
    r = mlp.get("router") or {}
    for k in ("experts", "top"):
        _positive(f"layer {i}: mlp.router.{k}", r.get(k))
    if r["top"] > r["experts"]:
        raise ConfigError(f"layer {i}: mlp.router.top {r['top']} is more than {r['experts']} experts")


@dataclass(frozen=True)
class GikaraxConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple                  # the ``layers`` list of config.json, each right half with decay_rank filled in
    loop: Optional[tuple] = None   # (start, stop, times) or None
    max_positions: int = DEFAULT_MAX_POSITIONS
    architecture: str = "Gikarax"

    # ---- construction -----------------------------------------------------

    @classmethod
    def from_dict(cls, cfg: dict, decay_ranks=None) -> "GikaraxConfig":
        """``decay_ranks``: per layer the rank found in the checkpoint (or None)."""
        missing = [k for k in ("vocab", "width", "norm", "layers") if k not in cfg]
        if missing:
            raise ConfigError(f"config.json lacks required keys: {missing}")
        if not isinstance(cfg["norm"], dict) or "eps" not in cfg["norm"]:
            raise ConfigError("config.json: norm.eps is missing")
        layers = copy.deepcopy(list(cfg["layers"]))
        if not layers:
            raise ConfigError("config.json lists no layers")
        for i, layer in enumerate(layers):
            _check_layer(i, layer)
            if layer["type"] == "parallel":
                right = layer["mixer"]["right"]
                rank = None if decay_ranks is None else decay_ranks[i]
                if rank is None:
                    rank = right.get("decay_rank")
                if rank is None:
                    raise ConfigError(f"layer {i}: the rank of the decay map is not known: no checkpoint tensor "
                                      "to read it from and no right.decay_rank")
                right["decay_rank"] = _positive(f"layer {i}: right.decay_rank", int(rank))
        loop = cfg.get("loop")
        if loop is not None:
            for k in ("start", "stop", "times"):
                if not isinstance(loop.get(k), int) or isinstance(loop.get(k), bool):
                    raise ConfigError(f"loop.{k} must be an integer")
            if not (0 <= loop["start"] <= loop["stop"] <= len(layers)) or loop["times"] < 1:
                raise ConfigError(f"loop {loop!r} does not fit {len(layers)} layers")
            loop = (loop["start"], loop["stop"], loop["times"])
        out = cls(vocab=_positive("vocab", cfg["vocab"]), width=_positive("width", cfg["width"]),
                  norm_eps=float(cfg["norm"]["eps"]), layers=tuple(layers), loop=loop,
                  max_positions=_positive("max_positions", cfg.get("max_positions", DEFAULT_MAX_POSITIONS)),
                  architecture=str(cfg.get("architecture", "Gikarax")))
        if out.norm_eps <= 0:
            raise ConfigError("norm.eps must be positive")
        return out

    @classmethod
    def from_json(cls, model_dir) -> "GikaraxConfig":
        from ..weights.loader import read_header

        model_dir = Path(model_dir)
        cfg = json.loads((model_dir / "config.json").read_text())
        shapes = {}
        for f in sorted(model_dir.glob("*.safetensors")):
            for name, meta in read_header(f).items():
                shapes[name] = meta["shape"]
        ranks = []
        for i in range(len(cfg.get("layers", []))):
            shape = shapes.get(f"l{i}.mix.right.a1")
            ranks.append(int(shape[0]) if shape else None)
        return cls.from_dict(cfg, ranks)

    def to_dict(self) -> dict:
        """The config.json content that ``from_dict`` reads back unchanged."""
        out = {"architecture": self.architecture, "layers": copy.deepcopy(list(self.layers)),
               "loop": None if self.loop is None else dict(zip(("start", "stop", "times"), self.loop)),
               "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        return out

    def validate(self) -> None:
        GikaraxConfig.from_dict(self.to_dict())

    # ---- derived -----------------------------------------------------------

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def looped(self) -> bool:
        return self.loop is not None and self.loop[1] > self.loop[0]

    def layer_runs(self) -> list:
        """(layer, whether a pass of the loop starts in front of it) in the order the layers run."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, False) for i in range(n)]
        start, stop, times = self.loop
        runs = [(i, False) for i in range(start)]
        for _ in range(times):
            runs += [(i, i == start) for i in range(start, stop)]
        return runs + [(i, False) for i in range(stop, n)]

    def num_parameters(self) -> int:
        w = self.width
        n = 2 * self.vocab * w + w + (2 * w * w if self.looped else 0)
        for layer in self.layers:
            m = layer["mixer"]
            n += w
            if layer["type"] == "attention":
                q, kv = m["heads"] * m["dim"], m["kv_heads"] * (m["dim"] + m["vdim"])
                n += (q + kv + m["heads"] + m["heads"] * m["vdim"]) * w + 2 * m["dim"]
            elif layer["type"] == "parallel":
                left, right = m["left"], m["right"]
                qkv = left["heads"] * left["dim"] + left["kv_heads"] * (left["dim"] + left["vdim"])
                n += qkv * (w + 1) + (left["heads"] * left["vdim"] + 1) * w
                hd, he, rank = right["heads"] * right["dim"], right["heads"] * right["vdim"], right["decay_rank"]
                n += (2 * hd + 3 * he) * w + rank * (w + hd) + hd + right["vdim"] + 2 * w
            else:
                hd, he, c, r = m["heads"] * m["dim"], m["heads"] * m["vdim"], m["kv_rank"], m["q_rank"]
                n += (r + c + 2 * he) * w + r + c + hd * r + (hd + he) * c
            mlp = layer.get("mlp")
            if mlp is not None:
                n += mlp["router"]["experts"] * (2 * mlp["expert"]["ff"] + 1) * w
        return n

    # ---- the plan ------------------------------------------------------------

    def _mixer(self, i: int) -> PartSpec:
        layer, w, eps = self.layers[i], self.width, self.norm_eps
        p, m = f"l{i}.mix.", layer["mixer"]

        def rope(c: dict, how: str):
            rot = c.get("rot")
            if rot is None or not rot["dims"]:
                return None
            return PartSpec("rope", {"head_dim": c["dim"], "rotary_dim": rot["dims"], "theta": float(rot["base"]),
                                     how: rot.get("scaling")})

        def attention(prefix: str, c: dict, **more) -> PartSpec:
            return PartSpec("masked_attention", dict(
                prefix=prefix, hidden_size=w, num_heads=c["heads"], num_kv_heads=c["kv_heads"], head_dim=c["dim"],
                v_head_dim=c["vdim"], scale=float(c["scale"]), **more))

        if layer["type"] == "attention":
            return attention(p, m, position_encoding=rope(m, "scaling"), qk_norm_eps=eps, mask="window",
                             mask_size=m["mask"]["size"], sink_score=SINK_SCORE, gate="head",
                             softcap=None if m.get("softcap") is None else float(m["softcap"]))
        if layer["type"] == "parallel":
            right = m["right"]
            return PartSpec("parallel", dict(
                branches=[
                    attention(p + "left.", m["left"], position_encoding=rope(m["left"], "yarn"), bias=True, out_bias=True),
                    PartSpec("gated_linear_attention", dict(
                        prefix=p + "right.", hidden_size=w, num_heads=right["heads"], head_dim=right["dim"],
                        v_head_dim=right["vdim"], decay_rank=right["decay_rank"], tau=float(right["tau"]), norm_eps=eps))],
                scales=[BRANCH_SCALE, BRANCH_SCALE], hidden_size=w,
                branch_norms=[dict(name=p + "left.out", eps=eps), dict(name=p + "right.out", eps=eps)]))
        return PartSpec("latent_attention", dict(
            prefix=p, hidden_size=w, num_heads=m["heads"], head_dim=m["dim"], rot_dim=0, v_head_dim=m["vdim"],
            kv_rank=m["kv_rank"], q_rank=m["q_rank"], scale=float(m["scale"]), position_encoding=None, norm_eps=eps,
            gate=True))

    def plan(self) -> ModelPlan:
        w = self.width
        norm = dict(size=w, eps=self.norm_eps)
        layers = []
        for i, layer in enumerate(self.layers):
            mlp = layer.get("mlp")
            ff = PartSpec("none", {}) if mlp is None else PartSpec("routed_experts", dict(
                prefix=f"l{i}.mlp.", hidden_size=w, intermediate_size=mlp["expert"]["ff"],
                num_experts=mlp["router"]["experts"], top=mlp["router"]["top"], route_scale=1.0, weight_eps=0.0,
                activation="gelu", score="chosen_softmax", correction=False))
            layers.append(LayerSpec(
                block=PartSpec("parallel_f32_stream", {}), mixer=self._mixer(i), feed_forward=ff,
                mixer_norm=PartSpec("stream_layer_norm", dict(name=f"l{i}.norm1", **norm)),
                feed_forward_norm=PartSpec("none", {})))
        # every run of a layer has a cache of its own
        schedule = tuple(ScheduleEntry(layer=i, cache=n, writes_cache=True, enters=enters)
                         for n, (i, enters) in enumerate(self.layer_runs()))
        return ModelPlan(
            hidden_size=w, vocab_size=self.vocab,
            embedding=PartSpec("scaled_token_embedding", dict(name="embed", vocab_size=self.vocab, hidden_size=w,
                                                              scale=1.0)),
            head=PartSpec("linear_head", dict(name="head", vocab_size=self.vocab, hidden_size=w)),
            final_norm=PartSpec("stream_layer_norm", dict(name="final.norm", **norm)),
            layers=tuple(layers), schedule=schedule, max_positions=self.max_positions, eos_token_ids=(),
            # (nothing is looped: the entry's matrix, if stored, is not used)
            ignored_names=() if self.looped else ("loop.in",),
            stream_entry=PartSpec("mix_with_start", dict(name="loop.in", hidden_size=w)) if self.looped else None,
        )
