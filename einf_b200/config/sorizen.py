"""Typed configuration of the Sorizen decoder: latent attention with sliding windows, several
residual streams, dense and routed feed-forwards, layers that run with another layer's tensors.

``config.json`` carries ``architecture: "Sorizen"``, ``vocab``, ``width``, ``norm.eps``,
``embedding.scale``, ``streams`` and ``layers``, a list with one entry per layer: ``type``
(``latent_attention`` or ``latent_attention_2``), ``mixer`` (its sizes and constants), ``mlp``
(``{"kind": "dense", "ff": n}``, ``{"kind": "moe", "expert": {"ff": n}, "router": {"experts": E,
"top": k, "scale": s, "groups": {"count": c, "keep": k}}}``, or null for a layer without a
feed-forward) and, for a layer that has no tensors of its own, ``weights_of``: the layer whose tensors
it runs with (its cache is its own).

The embedding row is multiplied by ``embedding.scale`` and starts every one of ``streams`` residual
streams x_1 .. x_s.  A sublayer reads ``u = sum_s in[s] x_s``, gives ``y = sublayer(norm(u))``, and
``x_t <- sum_s mix[s, t] x_s + out[t] y`` for all streams at once; after the last layer the streams are
added up, normed and multiplied by an output matrix of the model's own.  Norms are layer norms with
weight and bias.

Both mixers are latent attention without a query latent: the first ``kv_rank`` rows of ``W_dkv h`` are
RMS-normed into the latent, the other ``rot_dim`` are a rotated key part shared by all heads;
neighbouring dimensions are rotated as pairs, at frequencies that ``rot.scaling`` stretches
(``factor``, ``original``, ``fast``, ``slow``: see the ``rope`` part's ``yarn`` scaling); ``mask.size`` keys
of sliding window.  ``latent_attention`` has a stored sink per head in the softmax's denominator,
``latent_attention_2`` a gate ``sigmoid(W_g h)`` per head on its output.

A dense feed-forward is ``down(gelu(up h))`` with the exact GELU.  A routed one scores experts by
``sigmoid(z)``, opens the ``groups.keep`` groups of neighbours whose two best scores have the largest sum,
takes the ``top`` best experts in them and weighs their outputs by their scores, divided by the
scores' sum and times ``router.scale``.

Checkpoint names are ``embed``, ``head``, ``final.norm``, ``l<i>.norm1|norm2``, ``l<i>.hc1|hc2.in|out|mix``,
``l<i>.mix.q|dkv|dkv.norm|uk|uv|o|sink|g``, ``l<i>.mlp.up|down``, ``l<i>.mlp.router``,
``l<i>.mlp.e<j>.gate|up|down``; a norm's bias has its weight's name with ``.b`` added.
"""
from __future__ import annotations

import dataclasses
import math
from typing import Any, ClassVar

from .base import ConfigError, ModelConfig
from .specs import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

#: the design's fixed number: what is added to the sum that the chosen experts' scores are divided by
SCORE_SUM_EPS = 1e-20

_LATENT_NAMES = {
    "q_proj.weight": "q", "kv_down.weight": "dkv", "kv_norm.weight": "dkv.norm", "k_up.weight": "uk",
    "v_up.weight": "uv", "o_proj.weight": "o", "sink": "sink", "head_gate.weight": "g",
}
_MIXERS = ("latent_attention", "latent_attention_2")


def _positive(where: str, value: Any) -> int:
    if not isinstance(value, int) or isinstance(value, bool) or value <= 0:
        raise ConfigError(f"{where} must be a positive integer, got {value!r}")
    return value


def _number(where: str, value: Any, positive: bool = False) -> float:
    if isinstance(value, bool) or not isinstance(value, (int, float)):
        raise ConfigError(f"{where} must be a number, got {value!r}")
    if positive and not value > 0:
        raise ConfigError(f"{where} must be positive, got {value!r}")
    return float(value)


def _require(where: str, data: Any, keys) -> None:
    if not isinstance(data, dict):
        raise ConfigError(f"{where} must be an object")
    missing = [key for key in keys if key not in data]
    if missing:
        raise ConfigError(f"{where} lacks {', '.join(missing)}")


def _check_mixer(where: str, m: Any) -> None:
    sizes = ("heads", "dim", "rot_dim", "vdim", "kv_rank")
    _require(where, m, sizes + ("scale", "rot"))
    for key in sizes:
        _positive(f"{where}.{key}", m[key])
    _number(f"{where}.scale", m["scale"])
    rot = m["rot"]
    _require(f"{where}.rot", rot, ("base", "dims"))
    dims = _positive(f"{where}.rot.dims", rot["dims"])
    if dims % 2 or dims != m["rot_dim"]:
        raise ConfigError(f"{where}.rot.dims must be even and equal rot_dim {m['rot_dim']}, got {dims}")
    _number(f"{where}.rot.base", rot["base"], positive=True)
    if rot.get("scaling") is not None:
        keys = ("factor", "original", "fast", "slow")
        _require(f"{where}.rot.scaling", rot["scaling"], keys)
        for key in keys:
            _number(f"{where}.rot.scaling.{key}", rot["scaling"][key], positive=True)
        if math.log(rot["base"]) == 0.0:
            raise ConfigError(f"{where}.rot.base must not be 1 where its frequencies are scaled")
    if m.get("mask") is not None:
        _require(f"{where}.mask", m["mask"], ("size",))
        _positive(f"{where}.mask.size", m["mask"]["size"])


def _check_mlp(where: str, mlp: Any) -> None:
    if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
        raise ConfigError(f"{where}.kind must be dense or moe, got {mlp!r}")
    if mlp["kind"] == "dense":
        _positive(f"{where}.ff", mlp.get("ff"))
        return
    _positive(f"{where}.expert.ff", (mlp.get("expert") or {}).get("ff"))
    router = mlp.get("router")
    _require(f"{where}.router", router, ("experts", "top"))
    experts, top = _positive(f"{where}.router.experts", router["experts"]), _positive(f"{where}.router.top", router["top"])
    _number(f"{where}.router.scale", router.get("scale", 1.0))
    open_experts = experts
    groups = router.get("groups")
    if groups is not None:
        _require(f"{where}.router.groups", groups, ("count", "keep"))
        count = _positive(f"{where}.router.groups.count", groups["count"])
        keep = _positive(f"{where}.router.groups.keep", groups["keep"])
        if experts % count or keep > count:
            raise ConfigError(f"{where}.router: {experts} experts do not form {count} equal groups of which {keep} are kept")
        open_experts = keep * (experts // count)
    if top > open_experts:
        raise ConfigError(f"{where}.router: top {top} exceeds the {open_experts} experts that can be chosen")


@dataclasses.dataclass(frozen=True)
class SorizenConfig(ModelConfig):
    architecture: ClassVar[str] = "Sorizen"

    vocab: int
    width: int
    layers: list
    norm: dict
    embedding: dict
    streams: int

    def validate(self) -> None:
        for key in ("vocab", "width", "streams"):
            _positive(key, getattr(self, key))
        _require("norm", self.norm, ("eps",))
        _number("norm.eps", self.norm["eps"], positive=True)
        _require("embedding", self.embedding, ("scale",))
        _number("embedding.scale", self.embedding["scale"])
        if not isinstance(self.layers, (list, tuple)) or not self.layers:
            raise ConfigError("layers must be a non-empty list")
        for index, layer in enumerate(self.layers):
            where = f"layers[{index}]"
            _require(where, layer, ("type", "mixer"))
            if layer["type"] not in _MIXERS:
                raise ConfigError(f"{where}.type must be {' or '.join(_MIXERS)}, got {layer['type']!r}")
            _check_mixer(f"{where}.mixer", layer["mixer"])
            if layer.get("mlp") is not None:
                _check_mlp(f"{where}.mlp", layer["mlp"])
        for index, layer in enumerate(self.layers):
            if layer.get("weights_of") is None:
                continue
            other = self.layers[self.owner(index)]
            if any(layer.get(key) != other.get(key) for key in ("type", "mixer", "mlp")):
                raise ConfigError(f"layers[{index}] runs with the tensors of layer {layer['weights_of']}, whose entry differs")

    def owner(self, index: int) -> int:
        """The layer whose tensors layer ``index`` runs with (itself, or at the end of its ``weights_of``)."""
        seen = set()
        while self.layers[index].get("weights_of") is not None:
            seen.add(index)
            other = self.layers[index]["weights_of"]
            if not isinstance(other, int) or isinstance(other, bool) or not 0 <= other < len(self.layers) or other in seen:
                raise ConfigError(f"layers[{index}].weights_of must name a layer with tensors, got {other!r}")
            index = other
        return index

    def to_dict(self) -> dict[str, Any]:
        data = {"architecture": self.architecture}
        data.update(dataclasses.asdict(self))
        return data

    @property
    def eps(self) -> float:
        return float(self.norm["eps"])

    @property
    def init_std(self) -> float:
        # random matrices that keep activations of order one, so that scores spread
        return float(self.width) ** -0.5

    # The part-by-part description --------------------------------------
    def _norm(self, name: str) -> PartSpec:
        return PartSpec("layernorm", {"size": self.width, "eps": self.eps,
                                      "tensor_names": {"weight": "", "bias": ".b"}}, name)

    def _connection(self, prefix: str) -> PartSpec:
        return PartSpec("hyper_connection", {"streams": self.streams,
                                             "tensor_names": {"read": "in", "write": "out", "mix": "mix"}}, prefix)

    def _mixer(self, kind: str, m: dict, prefix: str) -> PartSpec:
        rot = m["rot"]
        scaling = rot.get("scaling")
        return PartSpec(
            "latent_attention",
            {
                "hidden_size": self.width, "num_heads": m["heads"], "head_size": m["dim"], "rotary_size": m["rot_dim"],
                "value_head_size": m["vdim"], "kv_rank": m["kv_rank"], "q_rank": None, "scale": float(m["scale"]),
                "eps": self.eps, "window": (m.get("mask") or {}).get("size"),
                "sink": kind == "latent_attention", "head_gate": kind == "latent_attention_2",
                "position": PartSpec("rope", {
                    "rotary_dim": int(rot["dims"]), "theta": float(rot["base"]), "layout": "interleaved",
                    "scaling": None if scaling is None else {
                        "kind": "yarn", **{k: float(scaling[k]) for k in ("factor", "original", "fast", "slow")}},
                }),
                "tensor_names": _LATENT_NAMES,
            },
            prefix,
        )

    def _feed_forward(self, mlp: dict, prefix: str) -> PartSpec:
        if mlp["kind"] == "dense":
            return PartSpec(
                "dense_mlp",
                {"hidden_size": self.width, "intermediate_size": int(mlp["ff"]), "activation": "gelu",
                 "tensor_names": {"up_proj.weight": "up", "down_proj.weight": "down"}},
                prefix,
            )
        router, groups = mlp["router"], mlp["router"].get("groups")
        experts = int(router["experts"])
        names = {"router.weight": "router"}
        for e in range(experts):
            for local, stored in (("gate_proj", "gate"), ("up_proj", "up"), ("down_proj", "down")):
                names[f"experts.{e}.{local}.weight"] = f"e{e}.{stored}"
        return PartSpec(
            "routed_mlp",
            {
                "hidden_size": self.width, "intermediate_size": int(mlp["expert"]["ff"]), "num_experts": experts,
                "top_k": int(router["top"]), "score": "sigmoid", "renormalise": True, "renormalise_eps": SCORE_SUM_EPS,
                "weight_scale": float(router.get("scale", 1.0)), "weight_on": "output",
                "groups": None if groups is None else {"count": int(groups["count"]), "keep": int(groups["keep"]),
                                                       "best": 2},
                "tensor_names": names,
            },
            prefix,
        )

    def model_spec(self) -> ModelSpec:
        layers, place = [], {}
        for index, layer in enumerate(self.layers):
            if layer.get("weights_of") is not None:
                continue
            prefix = f"l{index}."
            parts = {
                "mixer_connection": self._connection(prefix + "hc1."),
                "mixer_norm": self._norm(prefix + "norm1"),
                "mixer": self._mixer(layer["type"], layer["mixer"], prefix + "mix."),
            }
            if layer.get("mlp") is not None:
                parts["feed_forward_connection"] = self._connection(prefix + "hc2.")
                parts["feed_forward_norm"] = self._norm(prefix + "norm2")
                parts["feed_forward"] = self._feed_forward(layer["mlp"], prefix + "mlp.")
            place[index] = len(layers)
            layers.append(LayerSpec("prenorm_hyper", parts))
        schedule = tuple(ScheduleEntry(place[self.owner(index)]) for index in range(len(self.layers)))
        return ModelSpec(
            hidden_size=self.width,
            vocab_size=self.vocab,
            embedding=PartSpec(
                "embedding",
                {"vocab_size": self.vocab, "hidden_size": self.width, "scale": float(self.embedding["scale"]),
                 "tensor_names": {"weight": "embed"}},
                "",
            ),
            layers=tuple(layers),
            schedule=schedule,
            final_norm=self._norm("final.norm"),
            head=PartSpec(
                "linear_head",
                {"vocab_size": self.vocab, "hidden_size": self.width, "tensor_names": {"weight": "head"}},
                "",
            ),
            streams=self.streams,
        )
