"""Norms fused with the residual add.  ``rmsnorm``:

``residual += pending; out = weight * residual * rsqrt(mean(residual^2) + eps)``,
all in 32-bit, rounded once into the activation type: the reference's
``fused_add_rmsnorm`` (``src/einf/executors/torch/fused_ops.py:41-68``; weight
initialised to ones, eps inside the root, ``qwen.py:125-132``).  With ``offset``
o in the spec the stored tensor w lies around zero and the weight is ``o + w``
(added once, in 32-bit, when the part is built).

``layernorm``: ``residual += pending; out = (residual - mean) / sqrt(variance + eps) * weight + bias`` with
the mean of the squared deviations as the variance, all in 32-bit.

Where a model has several residual streams (``parts/stream.py``) what is normalised is what a sublayer
reads of them; either norm serves there through its ``weight``, ``bias``, ``centre`` and ``eps``.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..config.specs import TensorSpec
from .base import Norm, register_part


@register_part("norm", "rmsnorm")
class RMSNorm(Norm):
    @classmethod
    def tensor_specs(cls, spec):
        return {"weight": TensorSpec((spec["size"],), "offset" if spec.get("offset") else "scale")}

    @classmethod
    def kernel_libraries(cls, spec, runtime):
        return ("pointwise",)

    #: no bias, and the mean is not taken off
    bias = None
    centre = False

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        self.size = int(spec["size"])
        self.eps = float(spec["eps"])
        self.weight = runtime.vector(tensors["weight"])
        if spec.get("offset"):
            self.weight = (self.weight + float(spec["offset"])).contiguous()

    #: ``forward`` takes the step's status word (``status=``), where a kernel with a bounded wait reports
    takes_status = True

    def forward(self, pending, residual, rows: Optional[torch.Tensor] = None, status: Optional[torch.Tensor] = None):
        count = rows.shape[0] if rows is not None else residual.shape[0]
        out = torch.empty((count, self.size), dtype=self.runtime.dtype, device=residual.device)
        ops.add_rmsnorm(pending, residual, self.weight, self.eps, out, rows, status)
        return out


@register_part("norm", "layernorm")
class LayerNorm(Norm):
    centre = True

    @classmethod
    def tensor_specs(cls, spec):
        return {"weight": TensorSpec((spec["size"],), "scale"), "bias": TensorSpec((spec["size"],), "offset")}

    @classmethod
    def kernel_libraries(cls, spec, runtime):
        return ("hyper",)

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        self.size = int(spec["size"])
        self.eps = float(spec["eps"])
        self.weight = runtime.vector(tensors["weight"])
        self.bias = runtime.vector(tensors["bias"])

    def forward(self, pending, residual, rows: Optional[torch.Tensor] = None):
        count = rows.shape[0] if rows is not None else residual.shape[0]
        out = torch.empty((count, self.size), dtype=self.runtime.dtype, device=residual.device)
        # one plain stream: what is pending is added to it as it is
        ops.hyper_norm(pending, residual, 1, None, None, None if rows is not None or pending is None else residual,
                       self.weight, self.bias, True, self.eps, out, rows)
        return out
