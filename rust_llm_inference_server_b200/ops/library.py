"""Loads the kernel library and declares the C signature of every exported launcher.

There is no fallback: if the library cannot be built or loaded, or no CUDA device is present, the
first op raises.  Launchers return 0, a cudaError_t (> 0) or a negative library code.
"""

from __future__ import annotations

import ctypes
import os
from ctypes import c_float, c_int, c_longlong, c_void_p

from . import build

_lib = None

P = c_void_p
I = c_int
F = c_float
LL = c_longlong

# name -> argument types (the stream is always last)
SIGNATURES = {
    "rlis_embedding": [P, P, P, I, I, I, F, I, P],
    "rlis_embedding_sink": [P, P, P, P, P, P, P, I, I, I, F, P],
    "rlis_logit_transform": [P, I, I, LL, F, F, P],
    "rlis_attention_prefill_tile": [],
    "rlis_rmsnorm": [P, P, P, P, P, P, I, I, F, I, P],
    "rlis_layer_norm": [P, P, P, P, P, P, I, I, F, I, P],
    "rlis_swiglu": [P, P, I, I, I, I, P],
    "rlis_gemm_f32_nt": [P, P, P, I, I, I, P],
    "rlis_gemm_f32_nt_batched": [P, P, P, I, I, I, LL, LL, LL, I, LL, LL, LL, P],
    "rlis_post_norm_residual": [P, P, P, P, P, P, P, I, I, F, F, F, I, P],
    "rlis_sum_norm": [P, P, F, P, P, F, P, F, P, P, I, I, F, F, I, P],
    "rlis_head_norm_gate": [P, P, P, LL, P, I, I, I, F, I, I, P],
    "rlis_gated_delta": [P, LL, I, I, I, P, P, P, P, LL, P, P, P, P, P, P, P, I, I, I, I, I, I, I, F, F, I, P],
    "rlis_channel_delta": [P, LL, I, I, P, LL, I, P, P, P, P, LL, P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, F, F, I, P],
    "rlis_state_space": [P, LL, I, I, P, P, P, P, P, P, LL, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, P],
    "rlis_conv_recurrence_state_floats": [I, I, I, I, I],
    "rlis_stream_mix": [P, LL, LL, I, P, P, P, P, P, P, I, F, F, P, P, P, P, P, I, I, I, P],
    "rlis_gate_group_norm": [P, P, LL, P, P, I, I, I, F, I, P],
    "rlis_act_norm": [P, LL, I, P, P, LL, P, LL, I, I, F, I, P],
    "rlis_bias_act": [P, P, P, LL, I, I, I, P],
    "rlis_latent_kv_store": [P, LL, P, P, P, P, P, I, I, I, I, F, F, I, P, P, P, I, P],
    "rlis_latent_q_rope": [P, LL, P, P, P, I, I, I, I, I, I, F, I, I, P],
    "rlis_attention_latent": [P, P, P, P, P, P, P, P, I, I, I, I, I, I, F, I, P, LL, I, P],
    "rlis_attention_latent_mma_takes": [I, I],
    "rlis_attention_latent_prefill": [P, I, P, P, P, P, I, P, P, P, I, I, I, I, I, F, I, P, LL, P],
    "rlis_attention_latent_decode": [P, I, P, P, P, P, P, P, P, P, I, I, I, I, I, I, F, I, I, I, P, LL, P],
    "rlis_attention_latent_decode_cluster": [],
    "rlis_per_head_small": [P, LL, LL, P, P, LL, LL, I, I, I, I, P],
    "rlis_latent_step": [P, LL, P, LL, P, P, P, P, P, P, P, I, I, I, I, I, I, F, F, P],
    "rlis_lightning_scan": [P, LL, I, I, I, P, P, P, P, P, P, I, I, I, I, I, P, I, P],
    "rlis_recurrence_inputs": [P, LL, I, I, I, P, I, I, I, I, P, I, P, F, I, P, P, I, P],
    "rlis_recurrence_scan_rows": [P, LL, I, I, I, P, P, P, P, P, P, I, I, I, I, P, I, F, P, P, I, P],
    "rlis_recurrence_scan": [P, LL, I, I, I, I, P, P, P, P, P, P, I, I, I, I, I, P],
    "rlis_qk_norm_store": [P, LL, I, I, I, P, P, F, P, LL, F, P, P, P, P, I, I, I, I, I, I, P, I, F, P, F, I, I, P, I, I, P],
    "rlis_qk_row_norm_store": [P, LL, I, I, I, P, P, F, P, P, P, P, I, I, I, I, I, I, I, P],
    "rlis_attention_bias": [P, P, P, P, P, I, P, LL, P, P, P, P, I, I, I, I, I, I, I, F, I, P, P, I, I, P],
    "rlis_attention_bias_mma_takes": [I, I],
    "rlis_attention_bias_prefill": [P, P, P, P, P, I, P, LL, P, I, P, P, P, I, I, I, I, I, I, F, I, P, P, I, P],
    "rlis_attention_bias_decode": [P, P, P, P, P, P, I, P, LL, P, P, P, P, I, I, I, I, I, I, I, F, I, I, P, P, I, P],
    "rlis_attention_difference": [P, P, P, P, P, LL, P, P, P, P, I, I, I, I, I, I, I, F, F, I, F, F, F, I, P],
    "rlis_attention_difference_prefill": [P, P, P, P, P, LL, P, I, P, P, P, I, I, I, I, I, I, I, I, F, F, I, F, F, F, P],
    "rlis_attention_difference_prefill_takes": [I, I, I],
    "rlis_attention_difference_decode": [P, P, P, P, P, P, LL, P, P, P, P, I, I, I, I, I, I, I, I, F, F, I, I, F, F, F, P],
    "rlis_attention_difference_decode_takes": [I, I, I, I, I],
    "rlis_attention_difference_decode_width": [I],
    "rlis_attention_difference_decode_cluster": [],
    "rlis_attention_difference_decode_resident": [I, I],
    "rlis_moe_route": [P, P, P, P, P, P, I, I, I, I, F, P, I, I, I, I, I, P],
    "rlis_moe_align": [P, P, P, P, I, I, I, I, P],
    "rlis_moe_gemm": [P, P, P, P, P, P, I, I, I, I, I, I, F, F, F, LL, I, I, P],
    "rlis_moe_gather_rows": [P, P, P, I, I, I, I, P],
    "rlis_gemm_tcgen05_grouped": [P, P, P, I, I, I, I, P, I, F, F, F, P],
    "rlis_moe_gemm_mma": [P, P, P, P, P, P, I, I, I, I, I, I, F, F, F, LL, I, P],
    "rlis_moe_mma_takes_tile": [I],
    "rlis_moe_combine": [P, P, P, P, P, P, I, I, I, P, P, I, I, P],
    "rlis_glu_act": [P, P, I, I, F, F, F, F, I, P, I, P],
    "rlis_rope_cache": [P, P, P, P, P, P, P, I, I, I, I, I, I, P],
    "rlis_attention_generic": [P, P, P, P, P, P, P, P, I, I, I, I, I, I, F, I, I, P],
    "rlis_attention_decode": [P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, F, I, I, I, P],
    "rlis_attention_decode_pages": [P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, F, I, I, I, P],
    "rlis_attention_decode_qkv": [P, P, P, P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, F, I, I, I, P],
    "rlis_attention_prefill": [P, P, P, P, P, I, P, P, P, I, I, I, I, I, F, I, I, P],
    "rlis_attention_prefill_tc": [P, P, P, P, P, I, P, P, P, I, I, I, I, I, I, I, F, I, I, I, P],
    "rlis_attention_prefill_tc_takes": [I, I, I, I],
    "rlis_repetition_penalty": [P, P, P, P, P, I, I, LL, P],
    "rlis_sample_rows": [P, P, P, I, I, LL, P],
    "rlis_sample_filtered": [P, P, P, I, I, LL, P],
    "rlis_nll_rows": [P, P, P, I, I, LL, P],
    "rlis_gemm_tcgen05": [P, P, P, I, I, I, I, P],
    "rlis_gemm_tcgen05_glu": [P, P, P, I, I, I, F, F, F, F, P, P],
    "rlis_stream_gemm_fused": [P, LL, P, P, I, I, I, I, I, P, P, I, I, F, P, P, P, P, F, P, P],
    "rlis_stream_gemm_streams": [P, LL, P, I, I, I, P, P, LL, LL, I, P, P, P, P, F, P, P, P, P],
    "rlis_take_errors": [P, P],
    "rlis_stream_gemm_timeline": [I],
    "rlis_stream_gemm_timeline_read": [P, P],
    "rlis_attention_decode_last_variant": [],
}

OPTIONAL_SIGNATURES: dict = {}


class KernelError(RuntimeError):
    pass


# Switches for measurements and tests; nothing in the engine sets one.  In the library
# (csrc/kernels/runtime_switches.cu): pdl, stream_ctas, stream_min_stages, decode_stages, decode_cluster,
# decode_tma, prefill_splits, gemm_pair, filtered_cluster.  In Python (ops/__init__.py): fuse_norms, prefill_tcgen05, stream_rows.
# `RLIS_DEBUG=name=value,name=value` in the environment sets them when the library is loaded.
PYTHON_SWITCHES: dict = {}


def debug_set(name: str, value: int) -> None:
    """Holds one of the kernels' own choices fixed (see the list above)."""
    if name in PYTHON_SWITCHES:
        PYTHON_SWITCHES[name](int(value))
        return
    if lib().rlis_debug_set(name.encode(), int(value)) != 0:
        raise KernelError(f"no debug switch {name!r}")


def lib():
    global _lib
    if _lib is None:
        path = build.build_kernels()
        try:
            handle = ctypes.CDLL(path)
        except OSError as e:
            raise KernelError(f"cannot load the CUDA kernel library {path}: {e}") from e
        for name, args in {**SIGNATURES, **OPTIONAL_SIGNATURES}.items():
            try:
                fn = getattr(handle, name)
            except AttributeError as e:
                raise KernelError(f"kernel library {path} lacks symbol {name}") from e
            fn.argtypes = args
            fn.restype = c_int
        for name in ("rlis_gemm_tcgen05_error", "rlis_stream_gemm_error", "rlis_attention_prefill_tc_error",
                     "rlis_attention_decode_error", "rlis_attention_difference_decode_error"):
            fn = getattr(handle, name)
            fn.argtypes = []
            fn.restype = c_int
        handle.rlis_debug_set.argtypes = [ctypes.c_char_p, c_int]
        handle.rlis_debug_set.restype = c_int
        _lib = handle
        for item in filter(None, os.environ.get("RLIS_DEBUG", "").split(",")):
            name, _, value = item.partition("=")
            debug_set(name.strip(), int(value))
    return _lib


_CUDA_ERRORS = {1: "invalid value", 2: "out of memory", 9: "invalid configuration",
                98: "invalid device function", 209: "no kernel image for this device",
                700: "illegal address", 715: "illegal instruction", 719: "launch failure"}


def check(code: int, name: str) -> None:
    if code == 0:
        return
    if code == -1:
        raise KernelError(f"{name}: this kernel does not take these sizes or this element type")
    if code < 0:
        raise KernelError(f"{name}: library error {code}")
    raise KernelError(f"{name}: CUDA error {code} ({_CUDA_ERRORS.get(code, 'see cudaError_t')})")
