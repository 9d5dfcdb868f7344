"""Arrangements of parts in one layer.

``prenorm``: ``h += mixer(norm1(h)); h += feed_forward(norm2(h))``.  The
residual stream ``h`` is a 32-bit tensor; a sublayer's output stays *pending*
until the next norm adds it, so each add is fused with the norm that follows
(``src/einf/executors/torch/qwen.py:526-563``).  ``prenorm_mixer`` has no feed-forward, ``parallel``
feeds mixer and feed-forward from one norm, ``prenorm_stream`` adds a residual multiplier,
convolutions in front of the sublayers, a per-layer token input and a weighted sum over the depth,
``prenorm_hyper`` reads and writes several residual streams through vectors and matrices of its own.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from .base import CacheView, Part, StepContext, build_part, join_needs, part_class, register_part
from .stream import NormedPending


class Block(Part):
    mixer: Part
    #: ``forward`` takes a :class:`~einf_b200.parts.stream.NormedPending` as what is pending
    takes_normed_pending = False

    @classmethod
    def part_categories(cls) -> dict[str, str]:
        """Role name in :class:`LayerSpec.parts` -> part category."""
        raise NotImplementedError

    def forward(
        self, residual: torch.Tensor, pending: Optional[torch.Tensor], ctx: StepContext, cache: CacheView
    ) -> torch.Tensor:
        """Consume ``pending`` into ``residual`` and return the new pending output."""
        raise NotImplementedError


@register_part("block", "prenorm")
class PreNormBlock(Block):
    @classmethod
    def part_categories(cls):
        return {
            "mixer_norm": "norm",
            "mixer": "mixer",
            "feed_forward_norm": "norm",
            "feed_forward": "feed_forward",
        }

    def __init__(self, layer_spec, tensors, runtime):
        self.runtime = runtime
        self.spec = layer_spec
        for role, category in self.part_categories().items():
            setattr(self, role, build_part(category, layer_spec.parts[role], tensors, runtime))

    @staticmethod
    def _normalise(norm, pending, residual, ctx):
        # a norm that declares ``takes_status`` gets the step's status word as well
        if getattr(norm, "takes_status", False):
            return norm.forward(pending, residual, status=ctx.status)
        return norm.forward(pending, residual)

    def forward(self, residual, pending, ctx, cache):
        x = self._normalise(self.mixer_norm, pending, residual, ctx)
        mixed = self.mixer.forward(x, ctx, cache)
        x = self._normalise(self.feed_forward_norm, mixed, residual, ctx)
        return self.feed_forward.forward(x, ctx)


@register_part("block", "prenorm_mixer")
class PreNormMixerBlock(PreNormBlock):
    """``h += mixer(norm1(h))`` and nothing else: a layer without a feed-forward."""

    @classmethod
    def part_categories(cls):
        return {"mixer_norm": "norm", "mixer": "mixer"}

    def forward(self, residual, pending, ctx, cache):
        x = self._normalise(self.mixer_norm, pending, residual, ctx)
        return self.mixer.forward(x, ctx, cache)


@register_part("block", "parallel")
class ParallelBlock(PreNormBlock):
    """``h += mixer(n) + feed_forward(n)`` with one norm ``n = norm(h)`` that both sublayers read.
    A feed-forward that takes an addend sums both in its last kernel, in 32-bit; otherwise the
    pending value is the stack of both as float32 terms, which the next norm adds up."""

    @classmethod
    def part_categories(cls):
        return {"mixer_norm": "norm", "mixer": "mixer", "feed_forward": "feed_forward"}

    def forward(self, residual, pending, ctx, cache):
        x = self._normalise(self.mixer_norm, pending, residual, ctx)
        mixed = self.mixer.forward(x, ctx, cache)
        if getattr(self.feed_forward, "takes_addend", False):
            return self.feed_forward.forward(x, ctx, add=mixed)   # its last kernel adds the two up
        terms = [mixed if mixed.dim() == 3 else mixed[None], self.feed_forward.forward(x, ctx)[None]]
        return torch.cat([term.to(torch.float32) for term in terms], dim=0)


def build_block(layer_spec, tensors, runtime) -> Block:
    return part_class("block", layer_spec.block)(layer_spec, tensors, runtime)


@register_part("block", "prenorm_stream")
class PreNormStreamBlock(Block):
    """``h += m mixer(c1(norm1(h))); h += m ff(c2(norm2(h)))`` with a residual multiplier m and, each
    optional: a norm behind a sublayer (``m norm(mixer(..))``; run in the launch that adds the sublayer's output
    to the stream), a short causal convolution ``c(x) = x + conv(x)`` in front of a sublayer (run in the
    launch of the norm before it, continued from and into the request's state row), no feed-forward,
    a per-layer token input added after the feed-forward, and a weighted sum over the results of
    all layers so far in place of the layer's own result.  With a weighted sum the layer's last kernel
    adds the pending sublayer output, the token input and the sum in one pass over the row, and the
    block hands nothing pending to the next one; without one, what the layer added last stays pending
    (:class:`~einf_b200.parts.stream.NormedPending`) until the next layer's first norm.  The block's
    state row holds the convolutions' inputs in front of whatever state its mixer keeps."""

    optional_roles = ("mixer_conv", "mixer_post_norm", "feed_forward_norm", "feed_forward_conv", "feed_forward",
                      "feed_forward_post_norm", "token_input", "depth_mix")

    takes_normed_pending = True

    @classmethod
    def part_categories(cls):
        return {
            "mixer_norm": "norm",
            "mixer_conv": "stream",
            "mixer": "mixer",
            "mixer_post_norm": "norm",
            "feed_forward_norm": "norm",
            "feed_forward_conv": "stream",
            "feed_forward": "feed_forward",
            "feed_forward_post_norm": "norm",
            "token_input": "stream",
            "depth_mix": "stream",
        }

    def __init__(self, layer_spec, tensors, runtime):
        self.runtime = runtime
        self.spec = layer_spec
        self.residual_mult = float(layer_spec.params.get("residual_mult", 1.0))
        for role, category in self.part_categories().items():
            part = None
            if role in layer_spec.parts:
                part = build_part(category, layer_spec.parts[role], tensors, runtime)
            elif role not in self.optional_roles:
                raise KeyError(f"a prenorm_stream layer needs the part {role!r}")
            setattr(self, role, part)
        if (self.feed_forward is None) != (self.feed_forward_norm is None):
            raise ValueError("a feed-forward and its norm come together")
        if self.feed_forward is None and self.feed_forward_conv is not None:
            raise ValueError("a convolution in front of a feed-forward that is not there")
        if self.feed_forward is None and self.feed_forward_post_norm is not None:
            raise ValueError("a norm behind a feed-forward that is not there")
        for norm in (self.mixer_norm, self.mixer_post_norm, self.feed_forward_norm, self.feed_forward_post_norm):
            if norm is not None and (norm.centre or norm.bias is not None):
                raise ValueError("a prenorm_stream layer has RMS norms without bias")
        needs = [conv.state_need() if conv is not None else None for conv in (self.mixer_conv, self.feed_forward_conv)]
        self._need, offsets = join_needs(*needs, self.mixer.cache_need())
        self._conv_offsets, self._mixer_offset = offsets[:2], offsets[2]

    def cache_need(self):
        return self._need

    def _conv_state(self, which: int, cache: CacheView):
        conv = (self.mixer_conv, self.feed_forward_conv)[which]
        if conv is None or conv.taps == 1:
            return None
        offset = self._conv_offsets[which]
        rows = cache.state[:, offset:offset + (conv.taps - 1) * conv.size]
        return rows.unflatten(1, (conv.taps - 1, conv.size))

    def _normalise(self, which: int, pending, scale, post, residual, ctx, cache):
        """Add ``scale`` times what is pending (through the norm ``post`` behind its sublayer, if there is one) and
        return what the next sublayer reads."""
        norm = (self.mixer_norm, self.feed_forward_norm)[which]
        conv = (self.mixer_conv, self.feed_forward_conv)[which]
        out = torch.empty(residual.shape, dtype=self.runtime.dtype, device=residual.device)
        if conv is None:
            ops.stream_norm(pending, scale, post, residual, self._constants(norm), out)
            return out
        if pending is not None and post is not None:
            ops.stream_norm(pending, scale, post, residual, None, None)
            pending = None
        ops.norm_conv(
            pending, scale, residual, norm.weight, norm.eps, conv.weight,
            self._conv_state(which, cache), ctx.seq_of_token, ctx.q_start, ctx.state_slots, out,
            single_tokens=ctx.decode_only,
        )
        return out

    @staticmethod
    def _constants(norm):
        return None if norm is None else (norm.weight, norm.eps)

    def _add_token_input(self, terms, post, residual, ctx):
        """The token input's two matrices as products, behind a kernel that adds the pending output; the token
        input itself stays pending."""
        side, tokens = self.token_input, residual.shape[0]
        x = torch.empty(residual.shape, dtype=self.runtime.dtype, device=residual.device)
        ops.stream_norm(terms, self.residual_mult, post, residual, None, x)
        product = ops.project(x, side.gate, ctx.status)
        g = torch.empty((tokens, side.size), dtype=self.runtime.dtype, device=residual.device)
        ops.side_gate(product, side.table, ctx.token_ids, g)
        return NormedPending([ops.project(g, side.proj_rows, ctx.status)], self.residual_mult, (side.norm, side.eps))

    def forward(self, residual, pending, ctx, cache):
        if pending is not None and not isinstance(pending, NormedPending):
            raise ValueError("a prenorm_stream layer follows one that left its output pending")
        depth = self.depth_mix
        history = None
        if depth is not None:
            if pending is not None:
                pending.settle(residual)
                pending = None
            history = depth.history(ctx, residual)
            if depth.index == 0:
                history[0].copy_(residual)      # the embedding output, before this layer changes the stream
        if pending is None:
            x = self._normalise(0, None, 1.0, None, residual, ctx, cache)
        else:
            x = self._normalise(0, pending.terms, pending.scale, pending.norm, residual, ctx, cache)
        view = cache
        if self._mixer_offset is not None:
            view = CacheView(cache.group, cache.k, cache.v, cache.state[:, self._mixer_offset:], cache.writes,
                             cache.page_size)
        terms = self.mixer.forward_terms(x, ctx, view) if hasattr(self.mixer, "forward_terms") \
            else [self.mixer.forward(x, ctx, view)]
        post = self._constants(self.mixer_post_norm)
        if self.feed_forward is not None:
            x = self._normalise(1, terms, self.residual_mult, post, residual, ctx, cache)
            terms, post = [self.feed_forward.forward(x, ctx)], self._constants(self.feed_forward_post_norm)
        if depth is None:
            if self.token_input is None:
                return NormedPending(terms, self.residual_mult, post)
            return self._add_token_input(terms, post, residual, ctx)
        if post is not None:
            ops.stream_norm(terms, self.residual_mult, post, residual, None, None)
            terms = None
        side = self.token_input
        ops.stream_tail(
            residual, terms, self.residual_mult, ctx.token_ids,
            None if side is None else (side.table, side.gate, side.proj, side.norm, side.eps),
            (history, depth.index, depth.weight),
        )
        return None


@register_part("block", "prenorm_hyper")
class PreNormHyperBlock(Block):
    """Mixer and feed-forward on several residual streams (:class:`~einf_b200.parts.stream.ResidualStreams`):
    each sublayer has a connection that says what it reads of the streams, how they mix and what its
    output adds to each; the feed-forward with its norm and connection is optional.  ``residual`` is the
    streams; the write of the sublayer that ran last stays pending until the next norm."""

    optional_roles = ("feed_forward_connection", "feed_forward_norm", "feed_forward")

    @classmethod
    def part_categories(cls):
        return {
            "mixer_connection": "stream",
            "mixer_norm": "norm",
            "mixer": "mixer",
            "feed_forward_connection": "stream",
            "feed_forward_norm": "norm",
            "feed_forward": "feed_forward",
        }

    def __init__(self, layer_spec, tensors, runtime):
        self.runtime = runtime
        self.spec = layer_spec
        for role, category in self.part_categories().items():
            part = None
            if role in layer_spec.parts:
                part = build_part(category, layer_spec.parts[role], tensors, runtime)
            elif role not in self.optional_roles:
                raise KeyError(f"a prenorm_hyper layer needs the part {role!r}")
            setattr(self, role, part)
        if len({part is None for part in (self.feed_forward, self.feed_forward_norm, self.feed_forward_connection)}) > 1:
            raise ValueError("a feed-forward, its norm and its connection come together")

    def forward(self, residual, pending, ctx, cache):
        x = residual.normalise(self.mixer_norm, pending, self.mixer_connection)
        pending = self.mixer.forward(x, ctx, cache)
        if self.feed_forward is None:
            return pending
        x = residual.normalise(self.feed_forward_norm, pending, self.feed_forward_connection)
        return self.feed_forward.forward(x, ctx)
