"""Feed-forwards.  ``gated_mlp``: ``down(act(gate(x)) * up(x))`` with SiLU or the tanh form of GELU, or with
both branches clamped (:class:`GateActivation`); ``dense_mlp``: ``down(act(up(x)))``
with the square of ReLU (``relu2``), GELU (the exact form or the tanh form), SiLU or ReLU.

Gate and up share one matrix product on the concatenated weight, gate rows
first (``src/einf/executors/torch/qwen.py:163-172,206-208``); the activation is
SiLU (``fused_ops.py:71-77``), the only one Qwen2 uses (``qwen.py:138-139``).
"""
from __future__ import annotations

import torch

from .. import ops
from ..config.specs import TensorSpec
from .base import FeedForward, register_part


class GateActivation:
    """What joins a gated feed-forward's two branches: the name of an activation of the gate, which
    multiplies the other branch, or ``{"kind": "clamped_swish", "limit": c, "slope": a, "up_shift": b}``: with
    ``g = min(gate, c)`` and ``u = clamp(up, -c, c)`` the product is ``g sigmoid(a g) (u + b)``."""

    def __init__(self, spec) -> None:
        constants = dict(spec) if not isinstance(spec, str) else {"kind": spec}
        self.kind = str(constants.pop("kind"))
        if self.kind not in ops.GATE_ACTIVATIONS:
            raise ValueError(f"a gated feed-forward knows the activations {sorted(ops.GATE_ACTIVATIONS)}, not {self.kind!r}")
        if self.kind == "clamped_swish":
            self.constants = {key: float(constants.pop(key)) for key in ("limit", "slope", "up_shift")}
            if not self.constants["limit"] > 0:
                raise ValueError(f"the limit of a clamped branch must be positive, got {self.constants['limit']}")
        else:
            self.constants = {}
        if constants:
            raise ValueError(f"the activation {self.kind!r} has no {', '.join(sorted(constants))}")

    def __call__(self, gate_up: torch.Tensor, out: torch.Tensor) -> None:
        if self.kind == "silu":
            ops.silu_mul(gate_up, out)
        else:
            ops.act_mul(gate_up, out, self.kind, **self.constants)


@register_part("feed_forward", "gated_mlp")
class GatedMLP(FeedForward):
    @classmethod
    def tensor_specs(cls, spec):
        hidden, inter = spec["hidden_size"], spec["intermediate_size"]
        return {
            "gate_proj.weight": TensorSpec((inter, hidden)),
            "up_proj.weight": TensorSpec((inter, hidden)),
            "down_proj.weight": TensorSpec((hidden, inter)),
        }

    @classmethod
    def kernel_libraries(cls, spec, runtime):
        return ("pointwise", "gemm_simt") + (("gemm_tcgen05",) if runtime.dtype == torch.bfloat16 else ())

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        self.activation = GateActivation(spec.get("activation", "silu"))
        self.hidden_size = int(spec["hidden_size"])
        self.intermediate_size = int(spec["intermediate_size"])
        gate, up = tensors["gate_proj.weight"], tensors["up_proj.weight"]
        if gate.dtype != up.dtype:
            gate, up = gate.to(torch.float32), up.to(torch.float32)
        self.gate_up_weight = runtime.matrix(torch.cat([gate, up], dim=0))
        self.down_weight = runtime.matrix(tensors["down_proj.weight"])

    def forward(self, x, ctx):
        tokens = x.shape[0]
        dtype, device = self.runtime.dtype, x.device
        gate_up = ops.project(x, self.gate_up_weight, ctx.status)   # [T, 2I], or split-K partial sums
        hidden = torch.empty((tokens, self.intermediate_size), dtype=dtype, device=device)
        self.activation(gate_up, hidden)
        return ops.project(hidden, self.down_weight, ctx.status)


@register_part("feed_forward", "dense_mlp")
class DenseMLP(FeedForward):
    """Two matrices and an activation between them, no gate."""

    @classmethod
    def tensor_specs(cls, spec):
        hidden, inter = spec["hidden_size"], spec["intermediate_size"]
        return {"up_proj.weight": TensorSpec((inter, hidden)), "down_proj.weight": TensorSpec((hidden, inter))}

    @classmethod
    def kernel_libraries(cls, spec, runtime):
        return ("pointwise", "gemm_simt") + (("gemm_tcgen05",) if runtime.dtype == torch.bfloat16 else ())

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        self.activation = str(spec.get("activation", "relu2"))
        if self.activation not in ops.ACTIVATIONS:
            raise ValueError(f"dense_mlp knows the activations {sorted(ops.ACTIVATIONS)}, not {self.activation!r}")
        self.intermediate_size = int(spec["intermediate_size"])
        self.up_weight = runtime.matrix(tensors["up_proj.weight"])
        self.down_weight = runtime.matrix(tensors["down_proj.weight"])

    def forward(self, x, ctx):
        up = ops.project(x, self.up_weight, ctx.status)   # [T, I], or split-K partial sums
        hidden = torch.empty((x.shape[0], self.intermediate_size), dtype=self.runtime.dtype, device=x.device)
        ops.activation(up, hidden, self.activation)
        return ops.project(hidden, self.down_weight, ctx.status)
