"""Typed configuration of the Kumudra decoder, read from ``config.json``.

Kumudra is a small hybrid decoder whose residual stream has several parts (hyper-connections,
:mod:`scratch_llm_b200.parts.hyper_connection`): each sublayer reads a weighted sum of them through
a layer norm without an offset, and its output goes to every part, times ``residual_mult``, while the
parts mix.  ``layers`` lists the layers, each with one of three mixers:

* ``parallel``: two mixers side by side on the same input with constant weights.  Left: grouped-query
  attention with biases, values of a size of their own, a rotation of halves on the first ``rot.dims``
  entries of a head with the frequency scaling of Llama 3.1, and a sliding window
  (:mod:`scratch_llm_b200.parts.attention`).  Right: time mixing with a bonus
  (:mod:`scratch_llm_b200.parts.time_mixing`);
* ``gla``: gated linear attention, one decay per key channel; ``lightning``: linear attention with
  one constant decay per head (:mod:`scratch_llm_b200.parts.linear_attention`).

The feed-forward (``mlp``, or null) is a dense SwiGLU or routed: sigmoid scores, the choice by score
plus correction, the weights the chosen scores over their sum, times ``router.scale``.  The layers
``loop.start`` to ``loop.stop - 1`` run ``loop.times`` times in a row with the same weights, every
run with a cache entry and state of its own.  The output matrix is the embedding table.

config.json::

    {"architecture": "Kumudra", "vocab": V, "width": d, "norm": {"eps": e}, "streams": s,
     "residual_mult": m, "embedding": {"scale": c}, "loop": {"start", "stop", "times"},
     "layers": [{"type": "parallel", "mixer": {
                   "left": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size"},
                            "rot": {"base", "dims", "scaling": {"factor", "low", "high",
                                                                "original"} | null}},
                   "right": {"heads", "dim"}, "left_scale", "right_scale"},
                 "mlp": {"kind": "dense", "ff"} | {"kind": "moe", "expert": {"ff"},
                         "router": {"experts", "top", "scale"}} | null},
                {"type": "gla", "mixer": {"heads", "dim", "vdim", "tau"}, "mlp": ...},
                {"type": "lightning", "mixer": {"heads", "dim", "vdim", "decay": [per head]},
                 "mlp": ...}, ...]}

Without ``streams`` the stream is one sum and there are no ``hc`` tensors; without ``mask`` the
attention sees every earlier key, without ``rot`` nothing is rotated.

Tensors: ``embed``, ``final.norm`` and per layer i ``l<i>.norm1``, ``l<i>.norm2``,
``l<i>.hc1.{in,out,mix}``, ``l<i>.hc2.*``, ``l<i>.mix.*`` (``parallel``: ``l<i>.mix.left.*`` and
``l<i>.mix.right.*``) and ``l<i>.mlp.*``.
"""

from __future__ import annotations

import copy
import math
from dataclasses import dataclass, field
from typing import Any, Mapping

from .spec import LayerSpec, ModelSpec, PartSpec, Run

#: the design has no longest position; this bounds the rotary tables and the block tables
#: (config.json may carry another bound as "max_position")
DEFAULT_MAX_POSITION = 1 << 17

MIXERS = ("parallel", "gla", "lightning")


def _positive_int(value: Any, what: str) -> int:
    if not isinstance(value, int) or isinstance(value, bool) or value < 1:
        raise ValueError(f"{what} must be a positive integer, got {value!r}")
    return value


def _number(value: Any, what: str) -> float:
    if isinstance(value, bool) or not isinstance(value, (int, float)) or not math.isfinite(value):
        raise ValueError(f"{what} must be a number, got {value!r}")
    return float(value)


def _positive(value: Any, what: str) -> float:
    if not _number(value, what) > 0:
        raise ValueError(f"{what} must be positive, got {value!r}")
    return float(value)


def _mapping(value: Any, what: str) -> Mapping[str, Any]:
    if not isinstance(value, Mapping):
        raise ValueError(f"{what} must be an object, got {value!r}")
    return value


@dataclass(frozen=True)
class KumudraConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[Mapping[str, Any], ...]
    streams: int | None = None
    residual_mult: float = 1.0
    embedding_scale: float = 1.0
    loop: Mapping[str, int] | None = None
    max_position: int = DEFAULT_MAX_POSITION
    raw: Mapping[str, Any] = field(default_factory=dict, compare=False, repr=False)

    architecture = "Kumudra"

    def __post_init__(self) -> None:
        _positive_int(self.vocab, "vocab")
        _positive_int(self.width, "width")
        _positive_int(self.max_position, "max_position")
        if self.streams is not None:
            _positive_int(self.streams, "streams")
        if _number(self.norm_eps, "norm.eps") < 0:
            raise ValueError(f"norm.eps must not be negative, got {self.norm_eps!r}")
        _number(self.residual_mult, "residual_mult")
        _number(self.embedding_scale, "embedding.scale")
        if not self.layers:
            raise ValueError("layers must list at least one layer")
        for i, layer in enumerate(self.layers):
            self._check_layer(i, layer)
        if self.loop is not None:
            start, stop = self.loop.get("start"), self.loop.get("stop")
            for key, v in (("start", start), ("stop", stop)):
                if not isinstance(v, int) or isinstance(v, bool) or not 0 <= v <= len(self.layers):
                    raise ValueError(f"loop.{key} must name a place among the layers, got {v!r}")
            if start > stop:
                raise ValueError(f"loop.start {start} is behind loop.stop {stop}")
            _positive_int(self.loop.get("times"), "loop.times")

    def _check_layer(self, i: int, layer: Mapping[str, Any]) -> None:
        kind = layer.get("type")
        if kind not in MIXERS:
            raise ValueError(f"layer {i}: type must be one of {', '.join(MIXERS)}, got {kind!r}")
        where = f"layer {i}: mixer"
        m = _mapping(layer.get("mixer"), where)
        if kind == "parallel":
            self._check_attention(f"{where}.left", _mapping(m.get("left"), f"{where}.left"))
            right = _mapping(m.get("right"), f"{where}.right")
            for key in ("heads", "dim"):
                _positive_int(right.get(key), f"{where}.right.{key}")
            for key in ("left_scale", "right_scale"):
                _number(m.get(key), f"{where}.{key}")
        else:
            for key in ("heads", "dim", "vdim"):
                _positive_int(m.get(key), f"{where}.{key}")
            if kind == "gla":
                _positive(m.get("tau"), f"{where}.tau")
            else:
                decay = m.get("decay")
                if not isinstance(decay, (list, tuple)) or len(decay) != m["heads"] or \
                        not all(0.0 <= _number(a, f"{where}.decay") <= 1.0 for a in decay):
                    raise ValueError(f"{where}.decay must give one number from 0 to 1 per head, "
                                     f"got {decay!r}")
        self._check_feed_forward(f"layer {i}: mlp", layer.get("mlp"))

    @staticmethod
    def _check_attention(where: str, m: Mapping[str, Any]) -> None:
        for key in ("heads", "kv_heads", "dim", "vdim"):
            _positive_int(m.get(key), f"{where}.{key}")
        if m["heads"] % m["kv_heads"]:
            raise ValueError(f"{where}: {m['heads']} heads do not group evenly over "
                             f"{m['kv_heads']} key/value heads")
        _number(m.get("scale"), f"{where}.scale")
        if m.get("mask") is not None:
            _positive_int(_mapping(m["mask"], f"{where}.mask").get("size"), f"{where}.mask.size")
        if m.get("rot") is None:
            return
        rot = _mapping(m["rot"], f"{where}.rot")
        _positive(rot.get("base"), f"{where}.rot.base")
        dims = _positive_int(rot.get("dims"), f"{where}.rot.dims")
        if dims % 2 or dims > m["dim"]:
            raise ValueError(f"{where}.rot.dims must be even and at most dim = {m['dim']}, got "
                             f"{dims}")
        if rot.get("scaling") is not None:
            scaling = _mapping(rot["scaling"], f"{where}.rot.scaling")
            for key in ("factor", "low", "high", "original"):
                _positive(scaling.get(key), f"{where}.rot.scaling.{key}")
            if scaling["low"] > scaling["high"]:
                raise ValueError(f"{where}.rot.scaling.low is larger than high")

    @staticmethod
    def _check_feed_forward(where: str, mlp: Any) -> None:
        if mlp is None:
            return
        kind = _mapping(mlp, where).get("kind")
        if kind == "dense":
            _positive_int(mlp.get("ff"), f"{where}.ff")
            return
        if kind != "moe":
            raise ValueError(f"{where}.kind must be 'dense' or 'moe', got {kind!r}")
        router = _mapping(mlp.get("router"), f"{where}.router")
        experts = _positive_int(router.get("experts"), f"{where}.router.experts")
        if _positive_int(router.get("top"), f"{where}.router.top") > experts:
            raise ValueError(f"{where}.router.top is larger than the number of experts")
        _number(router.get("scale"), f"{where}.router.scale")
        _positive_int(_mapping(mlp.get("expert"), f"{where}.expert").get("ff"),
                      f"{where}.expert.ff")

    # -- config.json ---------------------------------------------------------------------

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "KumudraConfig":
        missing = [k for k in ("vocab", "width", "norm", "layers") if k not in raw]
        if missing:
            raise ValueError(f"config.json lacks required keys: {', '.join(missing)}")
        given = lambda v, default: default if v is None else v  # noqa: E731
        loop = raw.get("loop")
        return cls(vocab=raw["vocab"], width=raw["width"],
                   norm_eps=_number((raw["norm"] or {}).get("eps"), "norm.eps"),
                   layers=tuple(copy.deepcopy(dict(layer)) for layer in raw["layers"]),
                   streams=raw.get("streams"),
                   residual_mult=given(raw.get("residual_mult"), 1.0),
                   embedding_scale=given((raw.get("embedding") or {}).get("scale"), 1.0),
                   loop=None if loop is None else dict(loop),
                   max_position=raw.get("max_position", DEFAULT_MAX_POSITION),
                   raw=copy.deepcopy(dict(raw)))

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab,
                               "width": self.width, "norm": {"eps": self.norm_eps},
                               "residual_mult": self.residual_mult,
                               "embedding": {"scale": self.embedding_scale},
                               "layers": [copy.deepcopy(dict(layer)) for layer in self.layers]}
        if self.streams is not None:
            out["streams"] = self.streams
        if self.loop is not None:
            out["loop"] = dict(self.loop)
        if self.max_position != DEFAULT_MAX_POSITION:
            out["max_position"] = self.max_position
        return out

    @property
    def vocab_size(self) -> int:
        return self.vocab

    # -- layers as data ------------------------------------------------------------------

    def _mixer(self, kind: str, m: Mapping[str, Any]) -> tuple[PartSpec, PartSpec]:
        if kind == "parallel":
            left, right, rot = m["left"], m["right"], m["left"].get("rot")
            attention = {"hidden_size": self.width, "n_heads": left["heads"],
                         "n_kv_heads": left["kv_heads"], "head_dim": left["dim"],
                         "value_dim": left["vdim"], "scale": float(left["scale"]), "bias": True,
                         "window": (left.get("mask") or {}).get("size"),
                         "names": {n: n for n in "qkvo"}}
            time_mixing = {"hidden_size": self.width, "n_heads": right["heads"],
                           "head_dim": right["dim"], "eps": self.norm_eps}
            position = PartSpec("none") if rot is None else PartSpec("rotary", {
                "head_dim": left["dim"] + left["dim"] % 2, "theta": float(rot["base"]),
                "max_position": self.max_position, "interleaved": False,
                "rot_dims": rot["dims"], "llama3": rot.get("scaling")})
            return (PartSpec("side_by_side", {
                        "left": {"kind": "gqa_attention", "args": attention},
                        "right": {"kind": "time_mixing", "args": time_mixing},
                        "left_scale": float(m["left_scale"]),
                        "right_scale": float(m["right_scale"])}), position)
        common = {"hidden_size": self.width, "n_heads": m["heads"], "key_dim": m["dim"],
                  "value_dim": m["vdim"], "eps": self.norm_eps}
        if kind == "gla":
            return (PartSpec("gated_linear_attention", {**common, "tau": float(m["tau"])}),
                    PartSpec("none"))
        return (PartSpec("lightning_attention", {**common, "decay": tuple(m["decay"])}),
                PartSpec("none"))

    def _feed_forward(self, mlp: Mapping[str, Any]) -> PartSpec:
        if mlp["kind"] == "dense":
            return PartSpec("swiglu", {"hidden_size": self.width, "intermediate_size": mlp["ff"],
                                       "names": {n: n for n in ("gate", "up", "down")}})
        router = mlp["router"]
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "expert_size": mlp["expert"]["ff"],
            "experts": router["experts"], "top": router["top"], "score": "sigmoid",
            "weight_scale": float(router["scale"])})

    def run_order(self) -> tuple[Run, ...]:
        """The layers in their run order; every run has a cache entry of its own."""
        n = len(self.layers)
        loop = self.loop or {"start": 0, "stop": 0, "times": 1}
        start, stop = loop["start"], loop["stop"]
        order = [*range(start), *(list(range(start, stop)) * loop["times"]), *range(stop, n)]
        return tuple(Run(layer=layer, cache=i) for i, layer in enumerate(order))

    def model_spec(self) -> ModelSpec:
        norm = PartSpec("layernorm", {"size": self.width, "eps": self.norm_eps, "name": "",
                                      "bias": False})
        streams = PartSpec("hyper_connection", {
            "streams": self.streams or 1, "residual_mult": float(self.residual_mult),
            "learned": self.streams is not None})
        layers = []
        for i, layer in enumerate(self.layers):
            mixer, position = self._mixer(layer["type"], layer["mixer"])
            parts = {"mixer": mixer, "mixer_norm": norm, "mixer_streams": streams,
                     "position": position}
            if layer.get("mlp") is not None:
                parts.update(feed_forward=self._feed_forward(layer["mlp"]), feed_forward_norm=norm,
                             feed_forward_streams=streams)
            layers.append(LayerSpec(f"l{i}", "hyper_connected", parts, {
                "mixer": "mix", "mixer_norm": "norm1", "mixer_streams": "hc1",
                "feed_forward": "mlp", "feed_forward_norm": "norm2",
                "feed_forward_streams": "hc2"}))
        return ModelSpec(
            hidden_size=self.width, vocab_size=self.vocab, max_position=self.max_position,
            layers=tuple(layers), order=self.run_order(), final_norm=norm, embed_name="embed",
            final_norm_name="final.norm", lm_head_name="lm_head", tie_embeddings=True,
            embedding_multiplier=float(self.embedding_scale), streams=self.streams or 1)
