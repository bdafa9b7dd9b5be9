"""Typed configuration of the Deganex decoder, read from ``config.json``.

Deganex is a small hybrid decoder.  A layer's mixer and its feed-forward run side by side, each
behind an RMS norm of its own of the same stream, ``x + (mixer(norm1(x)) + ff(norm2(x)))``.  The
embedded tokens receive a second vector for the pair (previous token, token)
(:mod:`scratch_llm_b200.parts.token_pairs`); the logits pass a tanh cap.  ``layers`` lists the
layers, each with one of three mixers:

* ``latent_attention``: queries without a latent, one cached latent and one rotated key part per
  token, a rotation of adjacent pairs and a sigmoid gate per output channel
  (:mod:`scratch_llm_b200.parts.latent_attention`);
* ``mlstm``: a matrix memory with exponential gates
  (:mod:`scratch_llm_b200.parts.matrix_memory`);
* ``mamba2``: a state-space recurrence behind a short convolution
  (:mod:`scratch_llm_b200.parts.state_space`).

The feed-forward (``mlp``, or null) is routed: every token's weights are a softmax over its chosen
experts' logits, and a shared expert is added through a gate of one number per token
(:mod:`scratch_llm_b200.parts.routed`).  A layer with ``weights_of: j`` runs layer j again, with a
cache entry or state of its own.

config.json::

    {"architecture": "Deganex", "vocab": V, "width": d, "norm": {"eps": e}, "logit_softcap": c,
     "embedding": {"bigram": {"buckets": B, "mul_prev": a, "mul_cur": b}},
     "layers": [{"type": "mamba2",
                 "mixer": {"heads", "vdim", "state", "groups", "conv", "norm_groups"},
                 "mlp": {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"},
                         "shared": {"ff"}} | null},
                {"type": "latent_attention",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "scale",
                           "rot": {"base", "dims"}}, "mlp": ...},
                {"type": "mlstm", "mixer": {"heads", "dim", "vdim", "gate_cap"}, "mlp": ...},
                {..., "weights_of": j}, ...]}

Tensors: ``embed``, ``bigram``, ``head``, ``final.norm`` and per layer i without ``weights_of``
``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*`` and
``l<i>.mlp.{router,e<j>.gate,e<j>.up,e<j>.down,shared.gate,shared.up,shared.down,shared.sg}``.
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

MIXERS = ("latent_attention", "mlstm", "mamba2")


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


@dataclass(frozen=True)
class DeganexConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[Mapping[str, Any], ...]
    bigram: Mapping[str, int] | None = None
    logit_softcap: float = 0.0
    max_position: int = DEFAULT_MAX_POSITION
    raw: Mapping[str, Any] = field(default_factory=dict, compare=False, repr=False)

    architecture = "Deganex"

    def __post_init__(self) -> None:
        _positive_int(self.vocab, "vocab")
        _positive_int(self.width, "width")
        _positive_int(self.max_position, "max_position")
        if _number(self.norm_eps, "norm.eps") < 0:
            raise ValueError(f"norm.eps must not be negative, got {self.norm_eps!r}")
        if _number(self.logit_softcap, "logit_softcap") < 0:
            raise ValueError(f"logit_softcap must not be negative, got {self.logit_softcap!r}")
        if self.bigram is not None:
            _positive_int(self.bigram.get("buckets"), "embedding.bigram.buckets")
            for key in ("mul_prev", "mul_cur"):
                v = self.bigram.get(key)
                if not isinstance(v, int) or isinstance(v, bool) or v < 0:
                    raise ValueError(f"embedding.bigram.{key} must be an integer and not "
                                     f"negative, got {v!r}")
        if not self.layers:
            raise ValueError("layers must list at least one layer")
        for i, layer in enumerate(self.layers):
            self._check_layer(i, layer)

    def _check_layer(self, i: int, layer: Mapping[str, Any]) -> None:
        kind, m = layer.get("type"), layer.get("mixer")
        if kind not in MIXERS:
            raise ValueError(f"layer {i}: type must be one of {', '.join(MIXERS)}, got {kind!r}")
        if not isinstance(m, Mapping):
            raise ValueError(f"layer {i}: 'mixer' must give the mixer's sizes")
        where = f"layer {i}: mixer"
        sizes = {"latent_attention": ("heads", "dim", "rot_dim", "vdim", "kv_rank"),
                 "mlstm": ("heads", "dim", "vdim"),
                 "mamba2": ("heads", "vdim", "state", "groups", "conv", "norm_groups")}[kind]
        for key in sizes:
            _positive_int(m.get(key), f"{where}.{key}")
        if kind == "latent_attention":
            _number(m.get("scale"), f"{where}.scale")
            rot = m.get("rot")
            if not isinstance(rot, Mapping):
                raise ValueError(f"{where}.rot must give the rotation's base and dims")
            _positive(rot.get("base"), f"{where}.rot.base")
            dims = _positive_int(rot.get("dims"), f"{where}.rot.dims")
            if dims % 2 or dims > m["rot_dim"]:
                raise ValueError(f"{where}.rot.dims must be even and at most rot_dim = "
                                 f"{m['rot_dim']}, got {dims}")
        elif kind == "mlstm":
            _positive(m.get("gate_cap"), f"{where}.gate_cap")
        else:
            if m["heads"] % m["groups"]:
                raise ValueError(f"{where}: {m['heads']} heads do not group evenly over "
                                 f"{m['groups']} groups")
            if (m["heads"] * m["vdim"]) % m["norm_groups"]:
                raise ValueError(f"{where}: {m['heads'] * m['vdim']} channels do not form "
                                 f"{m['norm_groups']} equal parts")
        self._check_feed_forward(f"layer {i}: mlp", layer.get("mlp"))
        src = layer.get("weights_of")
        if src is None:
            return
        if not isinstance(src, int) or isinstance(src, bool) or not 0 <= src < len(self.layers) \
                or src == i:
            raise ValueError(f"layer {i}: weights_of must name another layer, got {src!r}")
        other = self.layers[self.owner(i)]
        if any(other.get(key) != layer.get(key) for key in ("type", "mixer", "mlp")):
            raise ValueError(f"layer {i} uses layer {src}'s tensors but differs from it")

    def owner(self, i: int) -> int:
        """The layer whose tensors layer ``i`` uses."""
        seen = [i]
        while self.layers[seen[-1]].get("weights_of") is not None:
            seen.append(self.layers[seen[-1]]["weights_of"])
            if seen[-1] in seen[:-1] or not 0 <= seen[-1] < len(self.layers):
                raise ValueError(f"layer {i}: weights_of leads to no layer with tensors of its own")
        return seen[-1]

    @staticmethod
    def _check_feed_forward(where: str, mlp: Any) -> None:
        if mlp is None:
            return
        if not isinstance(mlp, Mapping) or mlp.get("kind") != "moe":
            raise ValueError(f"{where}.kind must be 'moe', got "
                             f"{mlp.get('kind') if isinstance(mlp, Mapping) else mlp!r}")
        router = mlp.get("router") or {}
        experts = _positive_int(router.get("experts"), f"{where}.router.experts")
        if _positive_int(router.get("top"), f"{where}.router.top") > experts:
            raise ValueError(f"{where}.router.top is larger than the number of experts")
        _positive_int((mlp.get("expert") or {}).get("ff"), f"{where}.expert.ff")
        if mlp.get("shared") is not None:
            _positive_int(mlp["shared"].get("ff"), f"{where}.shared.ff")

    # -- config.json ---------------------------------------------------------------------

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "DeganexConfig":
        missing = [k for k in ("vocab", "width", "norm", "layers") if k not in raw]
        if missing:
            raise ValueError(f"config.json lacks required keys: {', '.join(missing)}")
        bigram = (raw.get("embedding") or {}).get("bigram")
        return cls(vocab=raw["vocab"], width=raw["width"],
                   norm_eps=_number((raw["norm"] or {}).get("eps"), "norm.eps"),
                   layers=tuple(copy.deepcopy(dict(layer)) for layer in raw["layers"]),
                   bigram=None if bigram is None else dict(bigram),
                   logit_softcap=raw.get("logit_softcap") or 0.0,
                   max_position=raw.get("max_position", DEFAULT_MAX_POSITION),
                   raw=copy.deepcopy(dict(raw)))

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab,
                               "width": self.width, "norm": {"eps": self.norm_eps},
                               "logit_softcap": self.logit_softcap,
                               "layers": [copy.deepcopy(dict(layer)) for layer in self.layers]}
        if self.bigram is not None:
            out["embedding"] = {"bigram": dict(self.bigram)}
        if self.max_position != DEFAULT_MAX_POSITION:
            out["max_position"] = self.max_position
        return out

    @property
    def vocab_size(self) -> int:
        return self.vocab

    # -- layers as data ------------------------------------------------------------------

    def _mixer(self, kind: str, m: Mapping[str, Any]) -> tuple[PartSpec, PartSpec]:
        common = {"hidden_size": self.width, "n_heads": m["heads"], "eps": self.norm_eps,
                  "value_dim": m["vdim"]}
        if kind == "latent_attention":
            return (PartSpec("latent_attention", {
                        **common, "dim": m["dim"], "rot_dim": m["rot_dim"], "q_rank": None,
                        "kv_rank": m["kv_rank"], "scale": float(m["scale"]), "gate": "wide",
                        "adjacent_pairs": m["rot"]["dims"]}),
                    PartSpec("rotary", {
                        "head_dim": m["rot_dim"] + m["rot_dim"] % 2,
                        "theta": float(m["rot"]["base"]), "max_position": self.max_position,
                        "interleaved": True, "rot_dims": m["rot"]["dims"]}))
        if kind == "mlstm":
            return (PartSpec("matrix_memory", {**common, "key_dim": m["dim"],
                                               "gate_cap": float(m["gate_cap"])}),
                    PartSpec("none"))
        return (PartSpec("state_space", {**common, "n_groups": m["groups"],
                                         "state_dim": m["state"], "conv_taps": m["conv"],
                                         "norm_groups": m["norm_groups"]}),
                PartSpec("none"))

    def _feed_forward(self, mlp: Mapping[str, Any]) -> PartSpec:
        shared = mlp.get("shared")
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "expert_size": mlp["expert"]["ff"],
            "experts": mlp["router"]["experts"], "top": mlp["router"]["top"],
            "correction": False, "shared_size": None if shared is None else shared["ff"],
            "shared_gate": shared is not None})

    def model_spec(self) -> ModelSpec:
        norm = PartSpec("rmsnorm", {"size": self.width, "eps": self.norm_eps, "name": ""})
        layers: list[LayerSpec] = []
        index: dict[int, int] = {}          # layer with tensors of its own -> its place in `layers`
        for i, layer in enumerate(self.layers):
            if layer.get("weights_of") is not None:
                continue
            mixer, position = self._mixer(layer["type"], layer["mixer"])
            parts = {"mixer": mixer, "mixer_norm": norm, "position": position}
            if layer.get("mlp") is not None:
                parts["feed_forward"] = self._feed_forward(layer["mlp"])
                parts["feed_forward_norm"] = norm
            index[i] = len(layers)
            layers.append(LayerSpec(f"l{i}", "parallel_norms", parts,
                                    {"mixer": "mix", "mixer_norm": "norm1",
                                     "feed_forward": "mlp", "feed_forward_norm": "norm2"}))
        order = tuple(Run(layer=index[self.owner(i)], cache=i) for i in range(len(self.layers)))
        pairs = None
        if self.bigram is not None:
            pairs = PartSpec("hashed_pairs", {"size": self.width, **{
                key: self.bigram[key] for key in ("buckets", "mul_prev", "mul_cur")}})
        return ModelSpec(
            hidden_size=self.width, vocab_size=self.vocab, max_position=self.max_position,
            layers=tuple(layers), order=order, final_norm=norm, embed_name="embed",
            final_norm_name="final.norm", lm_head_name="head", tie_embeddings=False,
            logit_softcap=float(self.logit_softcap), token_embedding=pairs,
            token_embedding_name="bigram")
