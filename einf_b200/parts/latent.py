"""Latent attention: keys and values of a token are one normed low-rank latent plus one rotated key
part that all heads share, and only those are cached.

Per token with input h: the query latent ``cq = rms(W_dq h) * w`` and the queries ``q = W_uq cq``, head by
head ``[dim plain | rot_dim rotated]``; ``W_dkv h`` gives the latent ``c = rms(first kv_rank) * w`` and the
key part ``r = rotate(last rot_dim)``.  Head h's key is ``[W_uk[h] c | r]``, its value ``W_uv[h] c``; scores
``(q_plain . k_plain + q_rot . r) * scale``, causal softmax, then the output projection.

Options, each from the spec: ``q_rank`` None, queries without a latent, ``q = W_q h`` (one product then gives
everything that h is projected to, and one kernel takes it apart); ``window``, the last that many keys
only; ``sink``, a stored number per head whose exponential joins the softmax's denominator, with no key and
no value; ``head_gate``, head h's mixed values are multiplied by ``sigmoid(W_g x)_h`` (in 32-bit, by the
attention kernel as it divides by the softmax's sum: the value up-projection is linear).

The cache holds the row ``[c | r]`` per token: one key/value head of size ``kv_rank + rot_dim`` whose first
``kv_rank`` elements double as the value.  The key up-projection is absorbed into the query
(``q_plain . W_uk[h] c = (W_uk[h]^T q_plain) . c``) and the value up-projection applied after the
mixing (``sum_j p_j W_uv[h] c_j = W_uv[h] sum_j p_j c_j``), so attention runs on the cached rows as they
are, with every query head on the one cached head.

In bfloat16 attention runs on the tensor cores wherever a cached row is a multiple of 64 elements, up to 640
(without a query latent other rows are filled up with zeros): ``ops.latent_attention``, a kernel of its own,
reads keys and values out of one tile.  Rows of 64 and 128 elements take the kernels of the attention mixer, with
the cached rows as keys and values at once: the mixed rows then carry ``rot_dim`` elements more than the value up-projection
reads (a fifth to a quarter more work in the second product, none in memory traffic).  Other row
sizes, and the 32-bit path, run the general kernel, which reads the values out of the key rows.
"""
from __future__ import annotations

import torch

from .. import ops
from ..config.specs import TensorSpec
from .base import CacheView, Mixer, PagedKVNeed, StepContext, build_nested, register_part


@register_part("mixer", "latent_attention")
class LatentAttention(Mixer):
    @classmethod
    def tensor_specs(cls, spec):
        hidden, heads = spec["hidden_size"], spec["num_heads"]
        dim, rot, value = spec["head_size"], spec["rotary_size"], spec["value_head_size"]
        kv_rank, q_rank = spec["kv_rank"], spec.get("q_rank")
        if q_rank:
            queries = {
                "q_down.weight": TensorSpec((q_rank, hidden)),
                "q_norm.weight": TensorSpec((q_rank,), "scale"),
                "q_up.weight": TensorSpec((heads * (dim + rot), q_rank)),
            }
        else:
            queries = {"q_proj.weight": TensorSpec((heads * (dim + rot), hidden))}
        if spec.get("sink"):
            queries["sink"] = TensorSpec((heads,), "bias")
        if spec.get("head_gate"):
            queries["head_gate.weight"] = TensorSpec((heads, hidden))
        return {
            **queries,
            "kv_down.weight": TensorSpec((kv_rank + rot, hidden)),
            "kv_norm.weight": TensorSpec((kv_rank,), "scale"),
            "k_up.weight": TensorSpec((heads * dim, kv_rank)),
            "v_up.weight": TensorSpec((heads * value, kv_rank)),
            "o_proj.weight": TensorSpec((hidden, heads * value)),
        }

    @classmethod
    def kernel_libraries(cls, spec, runtime):
        row = cls._row_size(spec, runtime.dtype)
        fast = ()
        if cls._row_on_tensor_cores(row, runtime.dtype):
            fast = (f"attention_tcgen05:HEAD_SIZE={row}",)
        elif ops.has_latent_attention(runtime.dtype, row, ops.LATENT_PAGE):
            fast = ("attention_latent",)
        return ("pointwise", "latent", "attention_generic", "gemm_simt") + \
            (("gemm_tcgen05",) if runtime.dtype == torch.bfloat16 else ()) + fast

    @staticmethod
    def _row_size(spec, dtype) -> int:
        """Elements of a cached row: latent and key part, and zeros up to a size the tensor-core kernels take."""
        row = int(spec["kv_rank"]) + int(spec["rotary_size"])
        filled = -(-row // ops.LATENT_ROW_MULTIPLE) * ops.LATENT_ROW_MULTIPLE
        if not spec.get("q_rank") and dtype == torch.bfloat16 and filled <= ops.MAX_GENERIC_HEAD_SIZE:
            return filled
        return row

    @staticmethod
    def _row_on_tensor_cores(row: int, dtype) -> bool:
        return dtype == torch.bfloat16 and row in (64, 128)

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        self.hidden_size = int(spec["hidden_size"])
        self.num_heads = int(spec["num_heads"])
        self.dim = int(spec["head_size"])
        self.rot_dim = int(spec["rotary_size"])
        self.value_size = int(spec["value_head_size"])
        self.kv_rank = int(spec["kv_rank"])
        self.q_rank = int(spec.get("q_rank") or 0)
        self.scale = float(spec["scale"])
        self.eps = float(spec["eps"])
        self.window = spec.get("window")
        if self.window is not None and self.window <= 0:
            raise ValueError(f"window must be positive, got {self.window}")
        self.row = self._row_size(spec, runtime.dtype)
        if self.row > ops.MAX_GENERIC_HEAD_SIZE:
            raise ops.UnsupportedSize(
                f"latent rows of {self.row} elements: the attention kernel takes up to {ops.MAX_GENERIC_HEAD_SIZE}")
        self.position = build_nested("position", spec["position"], tensors, runtime)
        if 2 * self.position.inv_freq.shape[0] != self.rot_dim:
            raise ValueError("the position encoding must rotate the whole rotated key part")
        heads = self.num_heads
        self.gated = bool(spec.get("head_gate"))
        if self.q_rank:
            if self.gated:
                raise ValueError("a gate per head comes with queries that have no latent")
            # one product for both down-projections: [query latent | kv latent | key part]
            rows = [tensors["q_down.weight"], tensors["kv_down.weight"]]
            self.q_norm = runtime.vector(tensors["q_norm.weight"])
            self.q_up = runtime.matrix(tensors["q_up.weight"])
        else:
            # one product for everything: [kv latent | key part | queries | gate logits]
            rows = [tensors["kv_down.weight"], tensors["q_proj.weight"]]
            if self.gated:
                rows.append(tensors["head_gate.weight"])
            # filled up so that a row of the product is a whole number of 16-byte pieces
            filled = -sum(m.shape[0] for m in rows) % 8
            if filled:
                rows.append(torch.zeros((filled, self.hidden_size), dtype=rows[0].dtype, device=rows[0].device))
        if len({m.dtype for m in rows}) > 1:
            rows = [m.to(torch.float32) for m in rows]
        self.down_weight = runtime.matrix(torch.cat(rows, dim=0))
        self.kv_norm = runtime.vector(tensors["kv_norm.weight"])
        self.sink = runtime.vector(tensors["sink"]) if spec.get("sink") else None
        # absorbed into the query: per head [kv_rank, dim], the transpose of the key up-projection
        k_up = tensors["k_up.weight"].reshape(heads, self.dim, self.kv_rank)
        self.k_up_t = runtime.matrix(k_up.transpose(1, 2).contiguous())
        self.v_up = runtime.matrix(tensors["v_up.weight"].reshape(heads, self.value_size, self.kv_rank))
        self.out_weight = runtime.matrix(tensors["o_proj.weight"])
        self.fast = self._row_on_tensor_cores(self.row, runtime.dtype)

    def launch_key(self, ctx: StepContext, page_size: int) -> tuple:
        """As for the attention mixer: the decode kernel's shape follows the batch and the longest context."""
        singles = int(ctx.single_tokens.shape[0])
        if not singles:
            return ()
        context = self._visible(ctx.max_context_len)
        if not self.fast and ops.has_latent_attention(self.runtime.dtype, self.row, page_size):
            return ("latent", ops.latent_attention_splits(singles, self.num_heads, self.kv_rank, context))
        if not (self.fast and ops.has_tcgen05_attention(self.row, page_size)):
            # the shared-row decode kernel cuts a token's keys by the batch and the longest context
            return ("shares", ops.latent_decode_splits(singles, self.num_heads, context)) if ctx.decode_only else ()
        return ops.decode_plan(singles, self.num_heads, 1, self.row, page_size, context)

    def _visible(self, context: int) -> int:
        return min(context, self.window) if self.window else context

    def launch_group(self):
        return ("latent_attention", self.num_heads, self.row, self.fast, self.window)

    def cache_need(self):
        # the values are the first kv_rank elements of the rows: no value cache of its own
        return PagedKVNeed(1, self.row, self.window, 0)

    def _queries_and_store(self, x, ctx: StepContext, cache: CacheView):
        """Project, write the step's cache rows, and return the queries' plain parts ``[T, H, dim]``, the full
        queries ``[T, H, row]`` with the rotated part in place, and the heads' gates."""
        tokens, heads, dim = x.shape[0], self.num_heads, self.dim
        dtype, device = self.runtime.dtype, x.device
        interleaved = getattr(self.position, "interleaved", False)
        amplitude = self.position.amplitude
        writes = cache.writes and cache.k is not None
        slots, pages = (ctx.slots[cache.group], cache.k) if writes else (None, None)
        q_full = torch.empty((tokens, heads, self.row), dtype=dtype, device=device)
        down = ops.project(x, self.down_weight, ctx.status)
        if not self.q_rank:
            gate = torch.empty((tokens, heads), dtype=torch.float32, device=device) if self.gated else None
            first, per_head = self.kv_rank + self.rot_dim, dim + self.rot_dim
            if down.dim() == 2 and down.dtype == dtype and first % 8 == 0 and per_head % 8 == 0:
                # the plain parts stay where the product left them (16-byte aligned rows)
                q_plain, copy = down[:, first:first + heads * per_head].unflatten(1, (heads, per_head))[..., :dim], None
            else:
                q_plain = copy = torch.empty((tokens, heads, dim), dtype=dtype, device=device)
            ops.latent_qkv_store(
                down, self.kv_rank, self.rot_dim, self.kv_norm, self.eps, ctx.positions, self.position.inv_freq,
                interleaved, amplitude, slots, copy, q_full, gate, pages, ctx.status, dim,
            )
            return q_plain, q_full, gate
        q_latent = torch.empty((tokens, self.q_rank), dtype=dtype, device=device)
        ops.latent_down_store(
            down, self.q_rank, self.kv_rank, self.rot_dim, self.q_norm, self.kv_norm, self.eps, ctx.positions,
            self.position.inv_freq, interleaved, slots, q_latent, pages, ctx.status, amplitude,
        )
        q = ops.project(q_latent, self.q_up, ctx.status)
        q_plain = torch.empty((tokens, heads, dim), dtype=dtype, device=device)
        ops.latent_q_store(q, ctx.positions, self.position.inv_freq, interleaved, q_plain, q_full, amplitude)
        return q_plain, q_full, None

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: CacheView) -> torch.Tensor:
        tokens = x.shape[0]
        dtype, device = self.runtime.dtype, x.device
        heads = self.num_heads
        q_plain, q_full, gate = self._queries_and_store(x, ctx, cache)
        ops.per_head_project(q_plain, self.k_up_t, q_full[:, :, : self.kv_rank])
        table = ctx.block_tables[cache.group]
        if self.fast and ops.has_tcgen05_attention(self.row, cache.k.shape[2]):
            # the cached rows are keys and values at once; the value up-projection reads the first kv_rank
            mixed_rows = torch.empty((tokens, heads, self.row), dtype=dtype, device=device)
            if ctx.single_tokens.shape[0]:
                ops.paged_decode_attention_auto(
                    q_full, cache.k, cache.k, table, ctx.seq_of_token, ctx.positions, mixed_rows, self.scale,
                    self.window, ctx.status, None if ctx.decode_only else ctx.single_tokens,
                    max_context=ctx.max_context_len, sink=self.sink, gate=gate,
                )
            if ctx.q_tiles.shape[0]:
                ops.paged_prefill_attention(
                    q_full, cache.k, cache.k, table, ctx.q_tiles, mixed_rows, self.scale, self.window, ctx.status,
                    cached_before=ctx.max_portion_start, sink=self.sink, gate=gate,
                )
            mixed_latent = mixed_rows[:, :, : self.kv_rank]
        elif ops.has_latent_attention(dtype, self.row, cache.k.shape[2]):
            mixed_latent = torch.empty((tokens, heads, self.kv_rank), dtype=dtype, device=device)
            ops.latent_attention(
                q_full, cache.k, table, ctx.seq_of_token, ctx.positions, ctx.q_tiles,
                None if ctx.decode_only else ctx.single_tokens, int(ctx.single_tokens.shape[0]), mixed_latent, self.scale,
                self.window, ctx.status, max_context=ctx.max_context_len, sink=self.sink, gate=gate,
            )
        elif ctx.decode_only:
            # every token stands alone: sixteen heads a CTA share the rows it stages, the keys are cut in shares
            mixed_latent = torch.empty((tokens, heads, self.kv_rank), dtype=dtype, device=device)
            ops.latent_decode_attention(
                q_full, cache.k, table, ctx.seq_of_token, ctx.positions, mixed_latent, self.scale,
                ops.latent_decode_splits(tokens, heads, self._visible(ctx.max_context_len)), ctx.status,
                self.window, self.sink, gate,
            )
        else:
            mixed_latent = torch.empty((tokens, heads, self.kv_rank), dtype=dtype, device=device)
            ops.paged_attention_generic(
                q_full, cache.k, None, table, ctx.seq_of_token, ctx.positions, mixed_latent,
                self.scale, self.window, ctx.status, values_in_keys=self.kv_rank, sink=self.sink, gate=gate,
            )
        mixed = torch.empty((tokens, heads, self.value_size), dtype=dtype, device=device)
        ops.per_head_project(mixed_latent, self.v_up, mixed)
        return ops.project(mixed.view(tokens, -1), self.out_weight, ctx.status)
