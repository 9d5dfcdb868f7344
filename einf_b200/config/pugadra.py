"""Typed configuration of the Pugadra decoder: windowed attention with convolved projections, norms on
both sides of every sublayer, clamped feed-forwards, a per-layer token input.

``config.json`` carries ``architecture: "Pugadra"``, ``vocab``, ``width``, ``norm.eps``,
``residual_mult``, ``token_side.dim`` and ``layers``, a list with one entry per layer: ``type``
(``attention``), ``mixer`` (its sizes and constants) and ``mlp`` (``{"kind": "dense", "ff": n, "limit": c}``,
``{"kind": "moe", "expert": {"ff": n, "limit": c}, "router": {"experts": E, "top": k}, "shared": {"ff": n,
"limit": c}}``, or null for a layer without a feed-forward).

With m the residual multiplier a layer computes ``x += m norm1b(mixer(norm1 x)); x += m norm2b(ff(norm2 x))``
with RMS norms whose stored weight lies around zero (the weight is one plus it), then adds its token
input: ``x += m rms(proj(gelu(gate x) * e)) w`` with e the layer's slice of a second embedding row of the
token and a plain weight w.  The output matrix is the embedding table.

The mixer is grouped-query softmax attention.  Queries, keys and values have biases and pass a causal
convolution over time of ``conv`` taps per channel; the first ``rot.dims`` dimensions of every query and key
head are rotated with neighbouring dimensions paired; a query sees the last ``mask.size`` keys; the
softmax's denominator holds one more than the sum of the exponentials (a sink of score zero); the heads
together are multiplied element by element by ``sigmoid(W_g h)`` and projected.  ``kv_from: j`` marks a
layer without key/value projections that reads the pages of layer j.

A feed-forward is ``down(g sigmoid(1.702 g) (u + 1))`` with ``g = min(gate h, limit)`` and ``u = clamp(up h, -limit,
limit)``.  A routed one takes the ``top`` experts with the largest logits ``W h + b``, weighs their outputs by
the softmax over the chosen logits, and adds a shared expert that every token takes.

Checkpoint names are ``embed``, ``side.embed``, ``l<i>.norm1|norm1b|norm2|norm2b``, ``l<i>.mix.q|k|v`` (each with
``.b`` and ``.conv``), ``l<i>.mix.g|o``, ``l<i>.mlp.gate|up|down``, ``l<i>.mlp.router|router.b``,
``l<i>.mlp.e<j>.gate|up|down``, ``l<i>.mlp.shared.gate|up|down``, ``l<i>.side.gate|proj|norm``, ``final.norm``.
"""
from __future__ import annotations

import dataclasses
from typing import Any, ClassVar, Optional

from .base import ConfigError, ModelConfig
from .specs import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

#: the design's fixed numbers: the factor inside the gate's sigmoid, what is added to the clamped other
#: branch, and the score of the softmax's sink
GATE_SLOPE = 1.702
UP_SHIFT = 1.0
SINK_SCORE = 0.0

_ATTENTION_NAMES = {
    "q_proj.weight": "q", "q_proj.bias": "q.b", "q_conv.weight": "q.conv",
    "k_proj.weight": "k", "k_proj.bias": "k.b", "k_conv.weight": "k.conv",
    "v_proj.weight": "v", "v_proj.bias": "v.b", "v_conv.weight": "v.conv",
    "gate_proj.weight": "g", "o_proj.weight": "o",
}
_MLP_NAMES = {"gate_proj.weight": "gate", "up_proj.weight": "up", "down_proj.weight": "down"}


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


def _check_mixer(where: str, m: Any, layers: list, index: int) -> None:
    sizes = ("heads", "kv_heads", "dim", "vdim", "conv")
    _require(where, m, sizes + ("scale",))
    for key in sizes:
        _positive(f"{where}.{key}", m[key])
    _number(f"{where}.scale", m["scale"])
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"{where}: {m['heads']} heads are not a multiple of {m['kv_heads']} kv_heads")
    rot = m.get("rot")
    if rot is not None:
        _require(f"{where}.rot", rot, ("base", "dims"))
        dims = _positive(f"{where}.rot.dims", rot["dims"])
        if dims % 2 or dims > m["dim"]:
            raise ConfigError(f"{where}.rot.dims must be even and at most {m['dim']}, got {dims}")
        _number(f"{where}.rot.base", rot["base"], positive=True)
    if m.get("mask") is not None:
        _require(f"{where}.mask", m["mask"], ("size",))
        _positive(f"{where}.mask.size", m["mask"]["size"])
    source = m.get("kv_from")
    if source is None:
        return
    if not isinstance(source, int) or isinstance(source, bool) or not 0 <= source < index:
        raise ConfigError(f"{where}.kv_from must name an earlier layer, got {source!r}")
    other = layers[source]["mixer"]
    if other.get("kv_from") is not None:
        raise ConfigError(f"{where}.kv_from names layer {source}, which has no keys of its own")
    if any(m.get(key) != other.get(key) for key in ("kv_heads", "dim", "vdim", "rot")):
        raise ConfigError(f"{where}.kv_from names layer {source}, whose key/value heads or rotation differ")


def _check_branch(where: str, data: Any) -> None:
    _require(where, data, ("ff", "limit"))
    _positive(f"{where}.ff", data["ff"])
    _number(f"{where}.limit", data["limit"], positive=True)


def _check_mlp(where: str, mlp: Any) -> None:
    if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
        raise ConfigError(f"{where}.kind must be dense or moe, got {mlp!r}")
    if mlp["kind"] == "dense":
        _check_branch(where, mlp)
        return
    _check_branch(f"{where}.expert", mlp.get("expert"))
    _require(f"{where}.router", mlp.get("router"), ("experts", "top"))
    experts = _positive(f"{where}.router.experts", mlp["router"]["experts"])
    if _positive(f"{where}.router.top", mlp["router"]["top"]) > experts:
        raise ConfigError(f"{where}.router: top {mlp['router']['top']} exceeds the {experts} experts")
    if mlp.get("shared") is not None:
        _check_branch(f"{where}.shared", mlp["shared"])


@dataclasses.dataclass(frozen=True)
class PugadraConfig(ModelConfig):
    architecture: ClassVar[str] = "Pugadra"

    vocab: int
    width: int
    layers: list
    norm: dict
    residual_mult: float = 1.0
    token_side: Optional[dict] = None

    def validate(self) -> None:
        for key in ("vocab", "width"):
            _positive(key, getattr(self, key))
        _require("norm", self.norm, ("eps",))
        _number("norm.eps", self.norm["eps"], positive=True)
        _number("residual_mult", self.residual_mult)
        if self.token_side is not None:
            _require("token_side", self.token_side, ("dim",))
            _positive("token_side.dim", self.token_side["dim"])
        if not isinstance(self.layers, (list, tuple)) or not self.layers:
            raise ConfigError("layers must be a non-empty list")
        for index, layer in enumerate(self.layers):
            where = f"layers[{index}]"
            _require(where, layer, ("type", "mixer"))
            if layer["type"] != "attention":
                raise ConfigError(f"{where}.type must be attention, got {layer['type']!r}")
            _check_mixer(f"{where}.mixer", layer["mixer"], self.layers, index)
            if layer.get("mlp") is not None:
                _check_mlp(f"{where}.mlp", layer["mlp"])

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
        return PartSpec("rmsnorm", {"size": self.width, "eps": self.eps, "offset": 1.0, "tensor_names": {"weight": ""}},
                        name)

    def _mixer(self, m: dict, prefix: str) -> PartSpec:
        rot = m.get("rot")
        position = PartSpec("none", {}) if rot is None else PartSpec(
            "rope", {"rotary_dim": int(rot["dims"]), "theta": float(rot["base"]), "layout": "interleaved"})
        return PartSpec(
            "attention",
            {
                "hidden_size": self.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"],
                "head_size": m["dim"], "value_head_size": m["vdim"], "qkv_bias": True, "out_bias": False,
                "scale": float(m["scale"]), "window": (m.get("mask") or {}).get("size"),
                "shared_kv": m.get("kv_from") is not None, "conv_taps": m["conv"], "sink_score": SINK_SCORE,
                "output_gate": True, "position": position, "tensor_names": _ATTENTION_NAMES,
            },
            prefix,
        )

    @staticmethod
    def _activation(limit: float) -> dict:
        return {"kind": "clamped_swish", "limit": float(limit), "slope": GATE_SLOPE, "up_shift": UP_SHIFT}

    def _feed_forward(self, mlp: dict, prefix: str) -> PartSpec:
        if mlp["kind"] == "dense":
            return PartSpec(
                "gated_mlp",
                {"hidden_size": self.width, "intermediate_size": int(mlp["ff"]),
                 "activation": self._activation(mlp["limit"]), "tensor_names": _MLP_NAMES},
                prefix,
            )
        experts, shared = int(mlp["router"]["experts"]), mlp.get("shared")
        names = {"router.weight": "router", "router.bias": "router.b"}
        for local, stored in _MLP_NAMES.items():
            names[f"shared.{local}"] = f"shared.{stored}"
            for e in range(experts):
                names[f"experts.{e}.{local}"] = f"e{e}.{stored}"
        return PartSpec(
            "routed_mlp",
            {
                "hidden_size": self.width, "intermediate_size": int(mlp["expert"]["ff"]), "num_experts": experts,
                # the softmax over the chosen logits is the softmax over all of them, divided by the chosen ones' sum
                "top_k": int(mlp["router"]["top"]), "score": "softmax", "renormalise": True, "weight_on": "output",
                "router_bias": True, "activation": self._activation(mlp["expert"]["limit"]),
                "shared": None if shared is None else int(shared["ff"]),
                "shared_activation": None if shared is None else self._activation(shared["limit"]),
                "tensor_names": names,
            },
            prefix,
        )

    def model_spec(self) -> ModelSpec:
        layers, schedule, unused = [], [], {}
        for index, layer in enumerate(self.layers):
            prefix = f"l{index}."
            parts = {
                "mixer_norm": self._norm(prefix + "norm1"),
                "mixer": self._mixer(layer["mixer"], prefix + "mix."),
                "mixer_post_norm": self._norm(prefix + "norm1b"),
            }
            if layer.get("mlp") is not None:
                parts["feed_forward_norm"] = self._norm(prefix + "norm2")
                parts["feed_forward"] = self._feed_forward(layer["mlp"], prefix + "mlp.")
                parts["feed_forward_post_norm"] = self._norm(prefix + "norm2b")
            else:       # the norms of a feed-forward that is not there
                unused.update({prefix + name: (self.width,) for name in ("norm2", "norm2b")})
            if self.token_side is not None:
                dim = int(self.token_side["dim"])
                parts["token_input"] = PartSpec(
                    "token_side_input",
                    {"hidden_size": self.width, "size": dim, "vocab_size": self.vocab,
                     "table_width": dim * len(self.layers), "table_offset": dim * index, "eps": self.eps,
                     "tensor_names": {"table": "side.embed", "gate.weight": prefix + "side.gate",
                                      "proj.weight": prefix + "side.proj", "norm.weight": prefix + "side.norm"}},
                    "",
                )
            layers.append(LayerSpec("prenorm_stream", parts, {"residual_mult": float(self.residual_mult)}))
            schedule.append(ScheduleEntry(index, layer["mixer"].get("kv_from")))
        return ModelSpec(
            hidden_size=self.width,
            vocab_size=self.vocab,
            embedding=PartSpec(
                "embedding", {"vocab_size": self.vocab, "hidden_size": self.width, "tensor_names": {"weight": "embed"}}, ""
            ),
            layers=tuple(layers),
            schedule=tuple(schedule),
            final_norm=self._norm("final.norm"),
            head=PartSpec(
                "linear_head",
                {"vocab_size": self.vocab, "hidden_size": self.width, "tied_to": "embed",
                 "tensor_names": {"weight": "head"}},
                "",
            ),
            unused_tensors=unused,
        )
