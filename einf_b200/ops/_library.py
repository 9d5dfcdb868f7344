"""Load the built kernel libraries through ctypes and bind their launchers."""
from __future__ import annotations

import ctypes
import threading
from typing import Sequence

from . import build

_libraries: dict[str, ctypes.CDLL] = {}
_lock = threading.Lock()

# Which source file holds which launcher.
LAUNCHERS = {
    "einf_embed": "pointwise",
    "einf_add_rmsnorm": "pointwise",
    "einf_rope_kv_write": "pointwise",
    "einf_silu_mul": "pointwise",
    "einf_advance_decode": "pointwise",
    "einf_add_bias": "pointwise",
    "einf_zero_fresh_state": "pointwise",
    "einf_activation": "pointwise",
    "einf_qkv_norm_store": "pointwise",
    "einf_conv_silu": "recurrence",
    "einf_linear_recurrence": "recurrence",
    "einf_gated_norm": "recurrence",
    "einf_paged_attention_generic": "attention_generic",
    "einf_latent_decode_attention": "attention_generic",
    "einf_latent_decode_merge": "attention_generic",
    "einf_latent_attention_tcgen05": "attention_latent",
    "einf_latent_attention_tcgen05_parts": "attention_latent",
    "einf_gemm_simt": "gemm_simt",
    "einf_gemm_tcgen05": "gemm_tcgen05",
    "einf_gemm_tcgen05_splits": "gemm_tcgen05",
    "einf_gemm_grouped_tcgen05": "gemm_tcgen05",
    "einf_paged_decode_attention": "attention_bf16",
    "einf_paged_decode_attention_cluster": "attention_bf16",
    "einf_paged_prefill_attention": "attention_bf16",
    "einf_paged_prefill_attention_tcgen05": "attention_tcgen05",
    "einf_paged_decode_attention_tcgen05": "attention_tcgen05",
    "einf_paged_prefill_attention_tcgen05_max_clusters": "attention_tcgen05",
    "einf_paged_decode_attention_tcgen05_max_clusters": "attention_tcgen05",
    "einf_latent_down_store": "latent",
    "einf_latent_q_store": "latent",
    "einf_latent_qkv_store": "latent",
    "einf_router_topk": "routed",
    "einf_moe_dispatch": "routed",
    "einf_moe_gemm": "routed",
    "einf_moe_combine": "routed",
    "einf_softcap": "pointwise",
    "einf_act_mul": "pointwise",
    "einf_norm_conv": "stream",
    "einf_stream_tail": "stream",
    "einf_stream_norm": "stream",
    "einf_side_gate": "stream",
    "einf_qkv_conv_store": "qkv_conv",
    "einf_hyper_norm": "hyper",
    "einf_paged_attention_mixed": "attention_mixed",
    "einf_paged_attention_mixed_tiled": "attention_mixed_tiled",
    "einf_paged_attention_mixed_tiled_rows": "attention_mixed_tiled",
    "einf_paged_attention_mixed_mma_ctas": "attention_mixed_tiled",
    "einf_gated_scan": "recurrence",
    "einf_memory_gates": "recurrence",
    "einf_memory_output": "recurrence",
    "einf_norm_join": "pointwise",
    "einf_argmax": "sampling",
    "einf_sample": "sampling",
    "einf_report": "sampling",
}


class KernelLibraryError(RuntimeError):
    """A kernel library could not be built or loaded: there is no fallback."""


def library(name: str) -> ctypes.CDLL:
    lib = _libraries.get(name)
    if lib is not None:
        return lib
    with _lock:
        lib = _libraries.get(name)
        if lib is None:
            try:
                path = build.build_kernel_library(name)
                lib = ctypes.CDLL(str(path))
            except (build.BuildError, OSError) as error:
                raise KernelLibraryError(
                    f"the CUDA kernel library '{name}' is not available and there is no "
                    f"fallback path: {error}"
                ) from error
            _libraries[name] = lib
    return lib


def ensure_built(names: Sequence[str]) -> None:
    """Compile the named libraries side by side and load them."""
    missing = [n for n in dict.fromkeys(names) if n not in _libraries]
    if not missing:
        return
    try:
        build.build_kernel_libraries(missing)
    except build.BuildError as error:
        raise KernelLibraryError(str(error)) from error
    for name in missing:
        library(name)


def launcher(symbol: str, argtypes: Sequence[type], variant: str = "") -> "ctypes._CFuncPtr":
    """Bind ``symbol``; ``variant`` (``MACRO=value``) picks a specialised build of its source."""
    source = LAUNCHERS[symbol] + (f":{variant}" if variant else "")
    function = getattr(library(source), symbol)
    function.argtypes = list(argtypes)
    function.restype = ctypes.c_int
    return function
