"""What a block does to the residual stream and to a sublayer's input besides norms.

``causal_conv_input``: what a sublayer reads, h, becomes ``h + conv(h)``: a causal convolution over
time on each channel, ``conv(h)_t = sum_j w[:, j] h_(t - taps + 1 + j)`` with zeros before the
sequence's start and no bias.  The last ``taps - 1`` inputs are per-request state (32-bit).  The
block runs it in the same launch as the norm in front of it.

``token_side_input``: a second embedding per token and layer.  ``e`` is the token's row of the
layer's slice of a table; ``g = gelu(W_gate x) * e`` with x the residual stream; ``y = W_proj g``;
the stream gets ``y / sqrt(mean(y^2) + eps) * w`` added (times the block's residual multiplier).

``depth_average``: with X_0 the embedding output and X_(i+1) the result of layer i, what leaves
layer i is ``sum_(j <= i + 1) w[j] X_j``.  The results of all layers of the step are kept in one
32-bit buffer in ``ctx.extras``.

The parts hold tensors and sizes; the block that arranges them (``prenorm_stream``) launches one
kernel for the end of a layer with a weighted sum: pending sublayer output, token input and sum together.
Without one the token input's matrices are two products with a kernel in front and between, and the
token input stays pending until the next layer's first norm (:class:`NormedPending`).

``hyper_connection``: the model has several residual streams x_1 .. x_s instead of one
(:class:`ResidualStreams`), all equal to the embedding output at the start.  A sublayer reads ``u = sum_s
read[s] x_s`` and, with y its output, every stream becomes ``x_t <- sum_s mix[s, t] x_s + write[t] y``.  The
write of one sublayer, what the next one reads and its norm are one launch (``ops.hyper_norm``), so
between sublayers y stays pending as it does for a single stream.
"""
from __future__ import annotations

import torch

from .. import ops
from ..config.specs import TensorSpec
from .base import Part, StateNeed, register_part


class NormedPending:
    """A pending output that enters the stream with a factor and, mostly, through a norm of its own: ``residual +=
    scale * rms(sum(terms)) * w`` with ``norm = (w, eps)``, or ``scale * sum(terms)`` (None).  A block that ``takes_normed_pending`` adds it in the launch of its first norm; in front
    of anything else it is settled by a launch of its own."""

    def __init__(self, terms, scale: float, norm) -> None:
        self.terms, self.scale, self.norm = terms, scale, norm

    def settle(self, residual: torch.Tensor) -> None:
        ops.stream_norm(self.terms, self.scale, self.norm, residual, None, None)


@register_part("stream", "causal_conv_input")
class CausalConvInput(Part):
    @classmethod
    def tensor_specs(cls, spec):
        return {"weight": TensorSpec((spec["size"], spec["taps"]), "conv")}

    @classmethod
    def kernel_libraries(cls, spec, runtime):
        return ("stream",)

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        self.size, self.taps = int(spec["size"]), int(spec["taps"])
        if not 1 <= self.taps <= ops.MAX_CONV_TAPS:
            raise ops.UnsupportedSize(f"{self.taps} taps: the convolution kernels take 1 to {ops.MAX_CONV_TAPS}")
        self.weight = runtime.vector(tensors["weight"])

    def state_need(self) -> StateNeed:
        """The last ``taps - 1`` inputs, oldest first, ``[taps - 1, size]`` floats in one row."""
        return StateNeed(((self.taps - 1) * self.size,), torch.float32)


@register_part("stream", "token_side_input")
class TokenSideInput(Part):
    @classmethod
    def tensor_specs(cls, spec):
        hidden, size = spec["hidden_size"], spec["size"]
        return {
            "table": TensorSpec((spec["vocab_size"], spec["table_width"])),
            "gate.weight": TensorSpec((size, hidden)),
            "proj.weight": TensorSpec((hidden, size)),
            "norm.weight": TensorSpec((hidden,), "scale"),
        }

    @classmethod
    def kernel_libraries(cls, spec, runtime):
        return ("stream", "gemm_simt") + (("gemm_tcgen05",) if runtime.dtype == torch.bfloat16 else ())

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        self.size = int(spec["size"])
        self.eps = float(spec["eps"])
        if self.size > ops.MAX_SIDE_SIZE:
            raise ops.UnsupportedSize(f"a token input of {self.size} values: the kernel takes up to {ops.MAX_SIDE_SIZE}")
        offset = int(spec.get("table_offset", 0))
        # this layer's columns of the table only: the layers together hold the table once
        self.table = runtime.matrix(tensors["table"][:, offset:offset + self.size].contiguous())
        self.gate = runtime.matrix(tensors["gate.weight"])
        self.proj_rows = runtime.matrix(tensors["proj.weight"])                 # [hidden, size], as a product takes it
        self.proj = self.proj_rows.t().contiguous()                             # [size, hidden]: rows are read along the stream
        self.norm = runtime.vector(tensors["norm.weight"])


@register_part("stream", "depth_average")
class DepthAverage(Part):
    @classmethod
    def tensor_specs(cls, spec):
        return {"weight": TensorSpec((spec["index"] + 2,), "depth")}

    @classmethod
    def kernel_libraries(cls, spec, runtime):
        return ("stream",)

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        self.index, self.layers = int(spec["index"]), int(spec["layers"])
        if not 0 <= self.index < self.layers:
            raise ValueError(f"layer {self.index} of {self.layers}")
        self.weight = runtime.vector(tensors["weight"])

    def history(self, ctx, residual: torch.Tensor) -> torch.Tensor:
        """The step's buffer ``[layers + 1, tokens, hidden]``: made by the first layer, which also puts
        the embedding output into its first row."""
        if self.index == 0:
            history = torch.empty((self.layers + 1, *residual.shape), dtype=torch.float32, device=residual.device)
            ctx.extras["depth_history"] = history
            return history
        history = ctx.extras.get("depth_history")
        if history is None or history.shape[1:] != residual.shape:
            raise RuntimeError("a depth average runs before the first layer of the step has made the history")
        return history


@register_part("stream", "hyper_connection")
class HyperConnection(Part):
    @classmethod
    def tensor_specs(cls, spec):
        streams = spec["streams"]
        return {
            "read": TensorSpec((streams,), "mean"),
            "write": TensorSpec((streams,), "scale"),
            "mix": TensorSpec((streams, streams), "near_identity"),
        }

    @classmethod
    def kernel_libraries(cls, spec, runtime):
        return ("hyper",)

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        self.streams = int(spec["streams"])
        if not 1 <= self.streams <= ops.MAX_STREAMS:
            raise ops.UnsupportedSize(f"{self.streams} residual streams: the kernel takes 1 to {ops.MAX_STREAMS}")
        self.read = runtime.vector(tensors["read"])
        self.write = runtime.vector(tensors["write"])
        self.mix = runtime.vector(tensors["mix"])       # [from, to]


class ResidualStreams:
    """The residual streams of a step, in the place of the one residual tensor: 32-bit ``[streams, T,
    hidden]``, or the one tensor ``[T, hidden]`` they all still equal before the first write.  The
    connection of the sublayer that ran last stays with them until its output, pending, is written."""

    def __init__(self, first: torch.Tensor, count: int) -> None:
        self.values, self.count = first, count
        self.connection: HyperConnection | None = None

    def normalise(self, norm, pending, connection=None, rows=None) -> torch.Tensor:
        """Write what is pending, and return the norm of what ``connection``'s sublayer reads (without
        one: of the sum of the streams) at all rows, or at ``rows``, for which nothing is stored."""
        before = self.connection
        if (pending is None) != (before is None):
            raise ValueError("a sublayer's output and its connection are written together")
        values = self.values
        tokens, hidden = values.shape[-2:]
        target = None
        if before is not None and rows is None:
            target = values if values.dim() == 3 else torch.empty((self.count, tokens, hidden), dtype=torch.float32,
                                                                  device=values.device)
        out = torch.empty((tokens if rows is None else rows.shape[0], hidden), dtype=norm.runtime.dtype,
                          device=values.device)
        ops.hyper_norm(
            pending, values, self.count, None if before is None else (before.mix, before.write),
            None if connection is None else connection.read, target, norm.weight, norm.bias, norm.centre, norm.eps,
            out, rows,
        )
        if target is not None:
            self.values = target
        self.connection = connection
        return out

    def total(self, pending) -> torch.Tensor:
        """The sum of the streams with what is pending written, ``[T, hidden]`` (for a look at the model
        from outside; the step itself never needs it)."""
        values = self.values if self.values.dim() == 3 else self.values.expand(self.count, *self.values.shape)
        if pending is None:
            return values.sum(0)
        y = (pending.sum(0) if pending.dim() == 3 else pending).float()
        return (self.connection.mix.sum(1)[:, None, None] * values).sum(0) + self.connection.write.sum() * y
