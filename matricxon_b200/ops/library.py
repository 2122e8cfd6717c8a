"""Loads the compiled kernel library and declares its C entry points.

There is no fallback: if the library cannot be built or loaded the error says so
and nothing runs (the reference's native ops instead decline by returning None,
app/native/fused_ops.py:130-230, and torch takes over; a GPU engine that fell
back silently would hide a missing build).
"""

from __future__ import annotations

import ctypes
import threading
from ctypes import c_float, c_int, c_longlong, c_void_p

from matricxon_b200.ops import build as _build


class KernelLibraryError(RuntimeError):
    pass


_lock = threading.Lock()
_lib: ctypes.CDLL | None = None

P, I, L, F = c_void_p, c_int, c_longlong, c_float

_SIGNATURES: dict[str, tuple[list, object]] = {
    "mx_last_error_message": ([], ctypes.c_char_p),
    "mx_set_chained_launch": ([I], None),
    "mx_embed": ([P, P, I, P, I, I, I, F, P, P], I),
    "mx_softcap": ([P, L, F, P], I),
    "mx_layernorm": ([P, P, P, P, P, I, I, I, F, P], I),
    "mx_layernorm_sum": ([P, P, P, P, P, P, I, I, I, F, P], I),
    "mx_rope_kv_write": ([P, I, I, P, P, P, P, I, I, I, I, I, I, L, I, P, P], I),
    "mx_rope_kv_write_bias": ([P, I, I, P, P, P, P, I, I, I, I, I, I, L, I, P, P, P], I),
    "mx_epilogue": ([P, I, P, P, P, I, L, I, I, P], I),
    "mx_gemm_simt": ([P, P, I, P, P, P, I, I, I, I, I, I, I, I, P], I),
    "mx_gemm_tcgen05": ([P, P, P, P, P, I, I, I, I, I, I, I, I, P, P], I),
    "mx_gemm_tcgen05_force_tiles": ([I], I),
    "mx_gemm_stream": ([P, P, P, P, P, I, I, I, I, I, I, I, I, P, P], I),
    "mx_gemm_skinny": ([P, P, P, P, P, I, I, I, I, I, I, I, I, P], I),
    "mx_gemm_skinny_rope": ([P, P, P, P, I, I, I, I, I, P, P, P, P, L, I, I, I, I, P, P], I),
    "mx_attention_scratch_bytes": ([I, I, I, I], L),
    "mx_paged_attention_mma": ([P, I, P, L, I, P, I, P, P, P, I, I, I, I, I, I, I, F, P, I, I, P, P, F, P, I, P, P], I),
    "mx_paged_attention_tc": ([P, I, P, L, I, P, I, P, P, P, I, I, I, I, I, I, F, P, I, P, P], I),
    "mx_paged_attention_tc_split": ([P, I, P, L, I, P, I, P, P, P, I, I, I, I, I, I, F, P, I, I, P, P, F, P, I, P, P], I),
    "mx_paged_attention": ([P, I, I, P, L, I, P, I, P, P, I, I, I, I, I, F, P, I, I, P, P, F, P, I, P, P], I),
    "mx_rmsnorm": ([P, P, P, F, P, I, I, I, F, L, P], I),
    "mx_add_row": ([P, P, I, I, P], I),
    "mx_rmsnorm_pending": ([P, P, P, P, F, P, I, I, I, F, P], I),
    "mx_rmsnorm_branch_add": ([P, P, P, P, P, I, I, I, F, P], I),
    "mx_rmsnorm_sum": ([P, P, F, P, F, P, I, I, I, F, P], I),
    "mx_cast_rows": ([P, P, L, P], I),
    "mx_cast_columns": ([P, I, P, I, I, P], I),
    "mx_latent_prepare": ([P, I, P, I, I, P, P, F, P, F, P, P, L, I, P, P, I, I, I, I, I, I, I, P, P], I),
    "mx_latent_attention_mma_supported": ([I, I], I),
    "mx_latent_attention_mma": ([P, P, L, I, P, I, P, P, P, I, I, I, I, I, I, I, F, P, I, P, I, P, P, P], I),
    "mx_latent_attention": ([P, P, I, L, I, P, I, P, P, I, I, I, I, I, F, P, P, P, P], I),
    "mx_qk_norm_kv_write": ([P, I, P, P, F, P, P, L, I, P, I, I, I, I, I, I, I, P, P], I),
    "mx_sigmoid_gate": ([P, P, I, P, I, I, I, I, I, P], I),
    "mx_clamped_glu": ([P, I, P, I, I, I, F, F, F, P], I),
    "mx_causal_conv": ([P, I, I, P, P, P, P, P, P, P, P, I, I, I, I, P], I),
    "mx_rglru_scan": ([P, I, I, I, P, P, P, P, F, P, P, P, P, I, I, I, I, I, P], I),
    "mx_rglru_scan_chunked": ([P, I, I, I, P, P, P, P, F, P, P, P, P, P, I, I, P, P, I, I, I, I, I, P], I),
    "mx_dyt": ([P, P, P, P, P, P, P, P, I, I, I, P], I),
    "mx_rotate_mix_kv_write": ([P, I, P, P, I, P, I, P, P, P, L, I, P, I, I, I, I, I, I, I, P, P], I),
    "mx_head_gate": ([P, P, I, P, I, I, I, I, I, P], I),
    "mx_gla_decay": ([P, I, P, P, F, P, I, I, I, P], I),
    "mx_gla_scan": ([P, I, I, I, I, P, F, P, P, P, P, I, I, I, I, P], I),
    "mx_retention_scan": ([P, I, I, I, I, P, F, P, P, P, P, I, I, I, I, P, P, I, I, P], I),
    "mx_retention_chunk_tokens": ([], I),
    "mx_retention_chunked": ([P, I, I, I, I, I, P, F, F, P, P, I, P, P, P, I, P, P, I, P, P, I, I, I, I, I, I, I, P], I),
    "mx_rotate_heads": ([P, I, I, I, I, I, I, P, P, P], I),
    "mx_conv_norm_kv_write": ([P, I, P, P, I, P, P, F, F, F, P, L, P, P, P, P, P, P, L, I, P, I, I, I, I, I, I, I, I, P, P], I),
    "mx_conv_state_update": ([P, I, I, P, P, L, P, P, I, I, I, P], I),
    "mx_conv_silu": ([P, I, I, P, P, P, L, P, P, P, P, I, I, I, I, P], I),
    "mx_selective_scan": ([P, P, I, P, I, P, P, P, P, I, I, P, L, L, P, P, P, I, I, I, I, I, I, F, P], I),
    "mx_selective_scan_chunked": ([P, P, I, P, I, P, P, P, P, I, I, P, L, L, P, P, P, I, I, I, I, I, I, F, P, P, I, I, P, P], I),
    "mx_selective_step": ([P, P, I, P, P, P, P, P, I, I, P, L, L, P, P, P, I, I, I, I, I, I, F, P], I),
    "mx_gla_norm_gate": ([P, P, I, P, F, P, I, I, I, I, I, I, F, I, P], I),
    "mx_norm_gate_rows": ([P, P, I, P, F, P, I, I, I, I, I, P], I),
    "mx_delta_prepare": ([P, I, I, I, P, I, P, P, P, L, P, P, P, P, P, P, I, I, I, I, I, F, F, P], I),
    "mx_delta_decay": ([P, I, P, P, P, P, I, I, I, I, P], I),
    "mx_delta_scan_scratch": ([I, I, I, I, I], L),
    "mx_delta_scan": ([P, P, P, I, P, L, L, P, P, P, P, P, I, I, I, I, I, I, P], I),
    "mx_delta_step": ([P, P, P, I, P, L, L, P, P, P, I, I, P, F, F, P, I, I, I, I, I, I, I, I, P], I),
    "mx_moe_route": ([P, I, I, P, I, I, I, I, I, F, I, P, P, P, P, I, P], I),
    "mx_moe_route_softmax": ([P, I, I, P, I, I, I, I, I, I, P, P, P, P, P, P, I, P], I),
    "mx_moe_tile_rows": ([], I),
    "mx_moe_plan": ([P, P, P, I, I, I, P, P, P, P, P], I),
    "mx_moe_gather": ([P, I, P, I, P, I, I, P], I),
    "mx_moe_combine_sorted": ([P, P, P, P, P, P, I, I, I, P, I, I, I, P], I),
    "mx_gemm_tcgen05_grouped": ([P, P, P, I, I, I, I, I, I, I, I, P, P, I, I, P, P], I),
    "mx_moe_gemm": ([P, I, I, P, I, P, L, I, I, P, P, I, P, P, I, I, F, F, F, P, P], I),
    "mx_moe_combine": ([P, P, I, I, I, P, P, P, I, I, I, P], I),
    "mx_rotate_norm_kv_write": ([P, I, P, P, I, F, P, P, L, I, P, I, I, I, I, I, I, I, P, P], I),
    "mx_norm_rotate_kv_write": ([P, I, P, P, I, I, F, P, P, F, P, P, L, I, P, I, I, I, I, I, I, I, I, F, P, P], I),
    "mx_layernorm_scaled_add": ([P, P, P, P, P, P, I, I, I, F, I, P], I),
    "mx_gelu_gate_rows": ([P, I, P, P, I, I, I, P, I, I, I, P, P], I),
    "mx_scale_rows": ([P, L, F, P], I),
    "mx_token_side_input": ([P, P, P, P, I, I, I, P, P, P, I, I, I, I, F, P, P], I),
    "mx_glu": ([P, I, P, I, I, I, I, P, P, P], I),
    "mx_gemm_batched_skinny": ([P, P, P, I, I, I, I, I, I, I, I, L, L, L, P], I),
    "mx_gemm_batched_simt": ([P, P, I, P, P, I, I, I, I, I, I, I, I, L, L, L, L, I, P], I),
}


def library() -> ctypes.CDLL:
    global _lib
    if _lib is not None:
        return _lib
    with _lock:
        if _lib is not None:
            return _lib
        try:
            path = _build.build()
        except _build.BuildError as exc:
            raise KernelLibraryError(
                f"the CUDA kernel library is missing and could not be built: {exc}") from exc
        try:
            lib = ctypes.CDLL(str(path))
        except OSError as exc:
            raise KernelLibraryError(f"cannot load {path}: {exc}") from exc
        for name, (argtypes, restype) in _SIGNATURES.items():
            try:
                fn = getattr(lib, name)
            except AttributeError as exc:
                raise KernelLibraryError(f"{path} lacks the entry point {name}") from exc
            fn.argtypes = argtypes
            fn.restype = restype
        _lib = lib
        return lib


def register_signature(name: str, argtypes: list, restype=c_int) -> None:
    """Declares one more entry point (kernel files added later list theirs here)."""
    _SIGNATURES[name] = (argtypes, restype)
    if _lib is not None:
        fn = getattr(_lib, name)
        fn.argtypes = argtypes
        fn.restype = restype


def check(code: int, what: str) -> None:
    if code == 0:
        return
    message = library().mx_last_error_message().decode("utf-8", "replace")
    if code == -1:
        raise KernelLibraryError(f"{what}: unsupported size: {message}")
    raise KernelLibraryError(f"{what}: failed with code {code}: {message}")
