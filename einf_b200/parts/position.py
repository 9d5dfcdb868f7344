"""Position encodings.  The attention mixer hands its raw QKV rows to the
position part, which adds the bias, encodes Q and K, and stores K and V in the
pages: one kernel does all three, so Q, K and V are read once.

``rope``: rotate-half rotary encoding over the first ``rotary_dim`` dims of each
head, ``inv_freq[i] = theta^(-2i/rotary_dim)``, angle ``position * inv_freq[i]``
in 32-bit (``src/einf/executors/torch/model_runner.py:42-78``).  The table of
inverse frequencies is made on the host by the reference's own expression, so
that angles agree with a host computation bit for bit.

With ``layout: "interleaved"`` pair i is dimensions (2i, 2i + 1) instead of (i, i + rotary_dim/2);
the general store kernel of the attention mixer rotates that layout.  With ``scaling`` (``factor``,
``low``, ``high``, ``original``) a frequency f of wavelength l = 2 pi / f stays as it is where
l < original / high, becomes f / factor where l > original / low, and between the two is
``(1 - s) f / factor + s f`` with ``s = (original / l - low) / (high - low)``: long wavelengths are
stretched, short ones kept.  ``scaling`` of ``kind: "yarn"`` (``factor``, ``original``, ``fast``, ``slow``) goes by
the pair's place instead: with ``dim(t) = rotary_dim * ln(original / (2 pi t)) / (2 ln theta)`` the pair that
turns t times over the original length, ``lo = max(floor(dim(fast)), 0)`` and ``hi = min(ceil(dim(slow)),
rotary_dim - 1)``, pair i keeps the share ``1 - r`` of its frequency and has the share r divided by
``factor``, ``r = clamp((i - lo) / max(hi - lo, 0.001), 0, 1)``; ``amplitude = 0.1 ln(factor) + 1`` then
multiplies cosine and sine (1 without this scaling; the latent mixer's kernels take it).

``none``: no encoding; bias and the cache write only.
"""
from __future__ import annotations

import math

import torch

from .. import ops
from .base import Part, register_part


class PositionEncoding(Part):
    def encode_and_store(self, qkv, bias, ctx, cache, q_out, num_heads, num_kv_heads, head_size):
        raise NotImplementedError


def _store(inv_freq, qkv, bias, ctx, cache, q_out, num_heads, num_kv_heads, head_size):
    writes = cache is not None and cache.writes and cache.k is not None
    ops.rope_kv_write(
        qkv,
        bias,
        ctx.positions,
        inv_freq,
        ctx.slots[cache.group] if writes else None,
        q_out,
        cache.k if writes else None,
        cache.v if writes else None,
        num_heads,
        num_kv_heads,
        head_size,
        ctx.status,
    )


@register_part("position", "rope")
class RotaryPosition(PositionEncoding):
    @classmethod
    def kernel_libraries(cls, spec, runtime):
        return ("pointwise",)

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        self.rotary_dim = int(spec["rotary_dim"])
        self.theta = float(spec["theta"])
        if self.rotary_dim % 2:
            raise ValueError(f"rotary_dim {self.rotary_dim} must be even")
        self.layout = str(spec.get("layout", "halves"))
        if self.layout not in ("halves", "interleaved"):
            raise ValueError(f"rotary layout must be halves or interleaved, got {self.layout!r}")
        self.interleaved = self.layout == "interleaved"
        scaling = spec.get("scaling")
        #: factor on cosine and sine
        self.amplitude = 1.0
        if scaling is None:
            inv_freq = 1.0 / (self.theta ** (torch.arange(0, self.rotary_dim, 2).float() / self.rotary_dim))
        elif scaling.get("kind") == "yarn":
            inv_freq = self.yarn_frequencies(self.theta, self.rotary_dim, scaling)
            self.amplitude = 0.1 * math.log(float(scaling["factor"])) + 1.0
        else:
            inv_freq = self.scaled_frequencies(self.theta, self.rotary_dim, scaling)
        self.inv_freq = inv_freq.to(runtime.device)

    @staticmethod
    def scaled_frequencies(theta: float, rotary_dim: int, scaling) -> torch.Tensor:
        """The frequency table with wavelength-dependent scaling, made in 64-bit on the host."""
        factor, low, high, original = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
        table = []
        for i in range(rotary_dim // 2):
            f = theta ** (-2.0 * i / rotary_dim)
            wavelength = 2.0 * math.pi / f
            if wavelength > original / low:
                f = f / factor
            elif wavelength >= original / high:
                blend = (original / wavelength - low) / (high - low)
                f = (1.0 - blend) * f / factor + blend * f
            table.append(f)
        return torch.tensor(table, dtype=torch.float64).to(torch.float32)

    @staticmethod
    def yarn_frequencies(theta: float, rotary_dim: int, scaling) -> torch.Tensor:
        """The frequency table with a ramp over the pairs, made in 64-bit on the host."""
        factor, original, fast, slow = (float(scaling[k]) for k in ("factor", "original", "fast", "slow"))

        def dim_of(turns: float) -> float:
            return rotary_dim * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(theta))

        low, high = max(math.floor(dim_of(fast)), 0), min(math.ceil(dim_of(slow)), rotary_dim - 1)
        table = []
        for i in range(rotary_dim // 2):
            f = theta ** (-2.0 * i / rotary_dim)
            ramp = min(max((i - low) / max(high - low, 0.001), 0.0), 1.0)
            table.append(f / factor * ramp + f * (1.0 - ramp))
        return torch.tensor(table, dtype=torch.float64).to(torch.float32)

    def encode_and_store(self, qkv, bias, ctx, cache, q_out, num_heads, num_kv_heads, head_size):
        if self.rotary_dim > head_size:
            raise ValueError(f"rotary_dim {self.rotary_dim} exceeds head size {head_size}")
        if self.amplitude != 1.0:
            raise ValueError("a factor on cosine and sine is taken by the latent mixer's kernels only")
        if self.interleaved:
            raise ValueError("the interleaved layout is rotated by the attention mixer's general store kernel")
        _store(self.inv_freq, qkv, bias, ctx, cache, q_out, num_heads, num_kv_heads, head_size)


@register_part("position", "none")
class NoPosition(PositionEncoding):
    @classmethod
    def kernel_libraries(cls, spec, runtime):
        return ("pointwise",)

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        self.inv_freq = torch.empty(0, dtype=torch.float32, device=runtime.device)
        self.amplitude = 1.0

    def encode_and_store(self, qkv, bias, ctx, cache, q_out, num_heads, num_kv_heads, head_size):
        _store(self.inv_freq, qkv, bias, ctx, cache, q_out, num_heads, num_kv_heads, head_size)
