"""Loads the compiled kernel library and declares its C functions.

There is no fallback: if the library cannot be built or loaded, or no CUDA
device is present, using a kernel raises `KernelLibraryError`.
"""
from __future__ import annotations

import ctypes
import threading
from ctypes import c_float, c_int, c_size_t, c_void_p

from . import build as _build


class KernelLibraryError(RuntimeError):
    pass


class KernelError(RuntimeError):
    """A kernel refused its arguments or failed to launch."""


_P = c_void_p
_I = c_int
_F = c_float

# name -> argument types (all return int)
_SIGNATURES = {
    "cuca_embed": [_P, _I, _P, _P, _I, _I, _I, _P, _P],
    "cuca_rmsnorm": [_P, _P, _I, _P, _I, _P, _I, _I, _F, _P],
    "cuca_rope_store": [_P, _I, _P, _P, _P, _I, _P, _P, _I, _I, _P, _P, _I, _I, _I, _I, _I, _I, _P, _P],
    "cuca_swiglu": [_P, _P, _I, _I, _I, _P],
    "cuca_add_to_stream": [_P, _P, _I, c_size_t, _P],
    "cuca_gemm_simt": [_P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _P],
    "cuca_attention_generic": [_P, _I, _P, _I, _I, _P, _P, _I, _I, _P, _P, _P, _I, _I, _I, _I, _I, _F, _I, _P, _P],
    "cuca_argmax": [_P, c_size_t, _I, _I, _P, _P],
    "cuca_suppress_tokens": [_P, c_size_t, _I, _I, _P, _I, _P],
    "cuca_scatter_int": [_P, _P, _P, _I, ctypes.c_longlong, _P],
    "cuca_sample": [_P, c_size_t, _I, _I, _P, _P, _P, _P, _P, _P, _P, _I, _P, _P, _I, _P],
    "cuca_sample_max_split": [],
    "cuca_attention_max_head_dim": [],
    "cuca_attention_mma_supported": [_I, _I, _I, _I, _I],
    "cuca_attention_decode": [_P, _I, _P, _I, _P, _P, _I, _I, _P, _P, _P, _I, _P, _I, _I, _I, _I, _F, _I, _I, _I,
                              _P, _P, _P, _P],
    "cuca_attention_decode_s": [_P, _I, _P, _I, _P, _P, _I, _I, _P, _P, _P, _I, _P, _I, _I, _I, _I, _F, _I, _F, _I, _I, _I,
                                _P, _P, _P, _P],
    "cuca_attention_decode_fused": [_P, _I, c_size_t, _P, _P, _P, _I, _I, _I, _P, _I, _P, _P, _I, _I, _P, _P, _P, _I,
                                    _P, _I, _I, _I, _I, _F, _I, _I, _I, _P, _P, _P, _P],
    "cuca_attention_prefill": [_P, _I, _P, _I, _P, _P, _I, _I, _P, _P, _P, _I, _P, _P, _I, _I, _I, _I, _F, _I, _P,
                               _P],
    "cuca_attention_prefill_s": [_P, _I, _P, _I, _P, _P, _I, _I, _P, _P, _P, _I, _P, _P, _I, _I, _I, _I, _F, _I, _F, _I, _P,
                                 _P],
    "cuca_decode_advance": [_P, _P, _P, _P, _P, _P, _I, _I, _P, _P, _P],
    "cuca_set_pdl": [_I],
    "cuca_attention_tc_supported": [_I, _I, _I, _I, _I, _I, _P, _P, _P],
    "cuca_attention_prefill_tc": [_P, _I, _I, _P, _I, _P, _P, _I, _I, _P, _P, _P, _I, _P, _P, _I, _I, _I, _I, _F, _I,
                                  _F, _I, _P, _P],
    "cuca_gemm_tc_glu": [_P, _P, _P, _I, _I, _I, _I, _I, _F, _F, _P, c_size_t, _P, _I, _I, _P, _P],
    "cuca_gemm_tc_partial_slices": [_I, _I, _I, _I],
    "cuca_gemm_tc_partial": [_P, _P, _P, _I, _I, _I, _I, _I, _P, _P, _P],
    "cuca_add_partials_rmsnorm": [_P, _P, _I, c_size_t, _P, _P, _I, _P, _I, _I, _F, _P],
    "cuca_add_partials": [_P, _P, _I, c_size_t, c_size_t, _P],
    "cuca_rope_store_partial": [_P, _I, c_size_t, _P, _P, _P, _P, _P, _I, _P, _P, _I, _I, _P, _P, _I, _I, _I, _I,
                                _I, _I, _P, _P],
    "cuca_sm_count": [],
    "cuca_gemm_tc_partial_max_tokens": [],
    "cuca_gemm_pair_mode": [_I],
    "cuca_attention_pair_tiles_mode": [_I],
    "cuca_gemm_tc_partial_rows": [_I, _I],
    "cuca_wait_probe": [ctypes.c_ulonglong, _P, _P, _P],
    "cuca_attention_tile_rows": [_I],
    "cuca_attention_plan": [_P, _P, _P, _I, _I, _P, _I, _P, _P, _I, _P],
    "cuca_random_normal": [_P, _I, c_size_t, c_size_t, ctypes.c_ulonglong, _F, _F, _P],
    "cuca_gemm_tc_supported": [_P, _P, _I, _I, _I, _I],
    "cuca_norm_shift": [_P, _P, _I, _F, _P, _P, _P, _I, _P, _P, _P, _P, _I, _I, _I, _P],
    "cuca_post_norm_add": [_P, _P, _P, _I, _P, _I, _P, _I, _I, _I, _F, _P],
    "cuca_gelu": [_P, _I, c_size_t, _I, _P],
    "cuca_scale": [_P, c_size_t, _F, _P],
    "cuca_concat2": [_P, _P, _P, _I, _I, _I, _P],
    "cuca_mingru_scan": [_P, _P, _P, _I, _P, _P, _P, _I, _I, _P],
    "cuca_mingru_scan_chunked": [_P, _P, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _P],
    "cuca_causal_conv": [_P, _I, _I, _P, _P, _I, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _P],
    "cuca_ssm_scan": [_P, _P, _I, _I, _P, _P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _P],
    "cuca_gated_group_norm": [_P, _P, _I, _P, _I, _P, _I, _I, _I, _I, _F, _P],
    "cuca_latent_max_rank": [],
    "cuca_latent_prepare": [_P, _I, _I, _I, _I, _I, _P, _F, _P, _P, _I, _I, _P, _P, _I, _I, _I, _P, _P, _P, _I, _I,
                            _P, _P],
    "cuca_head_linear": [_P, _I, _I, _P, _I, _P, _I, _I, _I, _P, _I, _I, _I, _I, _I, _P],
    "cuca_latent_attention": [_P, _P, _P, _I, _I, _I, _P, _P, _P, _I, _I, _I, _I, _I, _F, _I, _P, _P],
    "cuca_latent_attention_mma_supported": [_I, _I],
    "cuca_latent_attention_mma": [_P, _P, _P, _I, _I, _P, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _F, _I, _I, _P, _P,
                                  _P, _P],
    "cuca_attention_generic_v": [_P, _I, _P, _I, _I, _P, _P, _I, _I, _P, _P, _P, _I, _I, _I, _I, _I, _I, _F, _I, _P, _P],
    "cuca_rope_store_general": [_P, _I, _I, _I, _I, _P, _P, _P, _I, _P, _P, _I, _I, _I, _P, _P, _I, _I, _I, _I, _I, _I,
                                _I, _I, _I, _P, _P],
    "cuca_gate_merge": [_P, _P, _I, _P, _I, _I, _I, _I, _I, _P],
    "cuca_streams_max": [],
    "cuca_spread_streams": [_P, _P, _I, _I, _I, _P],
    "cuca_streams_read": [_P, _P, _P, _P, _I, _P, _I, _I, _I, _F, _P],
    "cuca_streams_write": [_P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _F, _P],
    "cuca_pair_norm_add": [_P, _P, _P, _P, _P, _F, _I, _I, _I, _F, _P],
    "cuca_sigmoid_gate": [_P, _I, _P, _I, _I, _I, _I, _P],
    "cuca_matrix_state_max_dim": [],
    "cuca_delta_scan": [_P, _I, _P, _I, _P, _P, _P, _I, _I, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _P],
    "cuca_mlstm_scan": [_P, _I, _I, _I, _I, _I, _I, _P, _P, _F, _P, _P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _P],
    "cuca_head_norm_gate": [_P, _P, _I, _P, _I, _I, _P, _I, _I, _I, _I, _F, _P],
    "cuca_moe_max_experts": [],
    "cuca_moe_route": [_P, _I, _I, _I, _P, _P, _P, _P],
    "cuca_moe_act_dense": [_P, _P, _P, _I, _I, _I, _I, _P],
    "cuca_moe_sparse": [_P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _I, _I, _P],
    "cuca_moe_route_scored": [_P, _P, _I, _I, _I, _I, _P, _P, _P, _P, _P],
    "cuca_moe_glu_dense": [_P, _P, _I, _P, _I, _I, _I, _I, _I, _P],
    "cuca_moe_identity_add": [_P, _P, _I, _P, _I, _I, _I, _P],
    "cuca_rmsnorm_groups": [_P, _P, _I, _P, _I, _P, _I, _I, _F, _I, _P],
    "cuca_add_partials_rmsnorm_groups": [_P, _P, _I, c_size_t, _P, _P, _I, _P, _I, _I, _F, _I, _P],
    "cuca_embed_scaled": [_P, _I, _P, _P, _I, _I, _I, _F, _P, _P],
    "cuca_glu_capped": [_P, _P, _I, _I, _I, _F, _F, _P],
    "cuca_attention_generic_s": [_P, _I, _P, _I, _I, _P, _P, _I, _I, _P, _P, _P, _I, _I, _I, _I, _I, _I, _F, _I, _F, _I,
                                 _P, _P],
    "cuca_norm_rope_store": [_P, _I, _I, _I, _I, _P, _I, _P, _P, _P, _I, _P, _P, _I, _I, _I, _P, _P, _I, _F, _P, _P, _I,
                             _I, _I, _I, _I, _I, _I, _I, _I, _P, _P],
    "cuca_forget_scan": [_P, _I, _I, _I, _I, _P, _P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _P],
    "cuca_gemm_tc": [_P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _P, c_size_t, _P, _I, _I, _P, _P],
    "cuca_gemm_tc_glu_act": [_P, _P, _P, _I, _I, _I, _I, _I, _I, _P, c_size_t, _P, _I, _I, _P, _P],
    "cuca_embed_norm": [_P, _I, _P, _P, _I, _I, _I, _F, _P, _F, _P, _P],
    "cuca_glu_act": [_P, _P, _I, _I, _I, _I, _P],
    "cuca_head_gate": [_P, _I, _P, _I, _I, _I, _I, _I, _P],
    "cuca_softcap": [_P, c_size_t, _F, _P],
    "cuca_attention_generic_sv": [_P, _I, _P, _I, _I, _P, _P, _I, _I, _P, _P, _P, _I, _I, _I, _I, _I, _I, _F, _I, _F, _I,
                                  _P, _P, _P],
    "cuca_attention_decode_sv": [_P, _I, _P, _I, _P, _P, _I, _I, _P, _P, _P, _I, _P, _I, _I, _I, _I, _F, _I, _F, _I, _P,
                                 _I, _I, _P, _P, _P, _P],
    "cuca_attention_prefill_sv": [_P, _I, _P, _I, _P, _P, _I, _I, _P, _P, _P, _I, _P, _P, _I, _I, _I, _I, _F, _I, _F, _I,
                                  _P, _P, _P],
    "cuca_attention_prefill_tc_sv": [_P, _I, _I, _P, _I, _P, _P, _I, _I, _P, _P, _P, _I, _P, _P, _I, _I, _I, _I, _F, _I,
                                     _F, _I, _P, _P, _P],
    "cuca_norm_rope_store_w": [_P, _I, _I, _I, _I, _P, _I, _P, _P, _P, _I, _P, _P, _I, _I, _I, _P, _P, _I, _F, _P, _P,
                               _I, _I, _I, _I, _I, _I, _I, _I, _I, _I, _F, _I, _P, _P],
    "cuca_latent_prepare_p": [_P, _I, _I, _I, _I, _I, _P, _F, _P, _P, _I, _I, _I, _P, _P, _I, _I, _I, _P, _P, _P, _I,
                              _I, _P, _P],
    "cuca_latent_attention_s": [_P, _P, _P, _I, _I, _I, _P, _P, _P, _I, _I, _I, _I, _I, _F, _I, _P, _P, _P],
    "cuca_latent_attention_mma_s": [_P, _P, _P, _I, _I, _P, _P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _F, _I, _P, _I, _P,
                                    _P, _P, _P],
    "cuca_retention_scan": [_P, _I, _I, _I, _I, _P, _P, _P, _I, _I, _F, _P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I,
                            _P, _P],
    "cuca_head_norm_gate_act": [_P, _P, _I, _P, _I, _I, _I, _P, _I, _I, _I, _I, _F, _P],
    "cuca_lightning_scan": [_P, _I, _I, _P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _P],
    "cuca_lightning_step": [_P, _I, _I, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _P],
    "cuca_max_terms": [],
    "cuca_norm_add": [_P, _P, _P, _P, _I, _I, _I, _F, _I, _P],
    "cuca_layer_norm": [_P, _P, _P, _I, _P, _I, _I, _F, _P],
    "cuca_add_terms": [_P, _P, _I, c_size_t, _P],
    "cuca_round_rows": [_P, _P, _I, c_size_t, _P],
    "cuca_row_norm_gate": [_P, _P, _P, _I, _I, _P, _I, _I, _I, _F, _P],
    "cuca_lightning_chunk_tokens": [],
    "cuca_lightning_chunk_max_dim": [],
    "cuca_lightning_chunked": [_P, _I, _I, _P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _P],
    "cuca_moe_sparse_act": [_P, _P, _P, _P, _P, _P, _I, _P, _I, _I, _I, _I, _I, _I, _I, _I, _I, _I, _I, _F, _F, _F, _P],
    "cuca_moe_route_grouped": [_P, _I, _I, _I, _I, _I, _F, _I, _P, _P, _P, _P],
    "cuca_moe_router_grouped": [_P, _P, _I, _I, _I, _I, _I, _I, _I, _F, _I, _P, _P, _P],
    "cuca_gemm_tc_glu_experts": [_P, _P, _P, _I, _I, _I, _I, _I, _F, _F, _F, _P, _I, _I, _I, _P, c_size_t, _P, _I, _I, _P,
                                 _P],
    "cuca_attention_generic_o": [_P, _I, _P, _I, _I, _P, _P, _I, _I, _P, _P, _P, _I, _I, _I, _I, _I, _I, _P, _P, _P],
    "cuca_attention_decode_o": [_P, _I, _P, _I, _P, _P, _I, _I, _P, _P, _P, _I, _P, _I, _I, _I, _I, _P, _I, _I, _P, _P, _P,
                                _P],
    "cuca_attention_prefill_o": [_P, _I, _P, _I, _P, _P, _I, _I, _P, _P, _P, _I, _P, _P, _I, _I, _I, _I, _P, _P, _P],
    "cuca_attention_prefill_tc_o": [_P, _I, _I, _P, _I, _P, _P, _I, _I, _P, _P, _P, _I, _P, _P, _I, _I, _I, _I, _P, _P, _P],
    "cuca_attention_decode_fused_unit": [_P, _I, c_size_t, _P, _I, _I, _I, _F, _P, _P, _I, _P, _P, _I, _I, _P, _P, _P, _I,
                                         _P, _I, _I, _I, _I, _P, _I, _I, _P, _P, _P, _P],
    "cuca_norm_rope_store_u": [_P, _I, _I, _I, _I, _P, _I, _P, _P, _P, _I, _P, _P, _I, _I, _I, _P, _P, _I, _F, _P, _P,
                               _I, _I, _I, _I, _I, _I, _I, _I, _I, _I, _F, _I, _I, _P, _P, _P, _P],
    "cuca_gemm_tc_act": [_P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _P, c_size_t, _P, _I, _I, _P, _P],
    "cuca_activation": [_P, _I, c_size_t, _I, _P],
    "cuca_embed_pos": [_P, _P, _I, _P, _P, _P, _I, _I, _I, _I, _F, _P, _P],
    "cuca_sum_norm": [_P, _P, _P, _P, _F, _F, _P, _I, _I, _I, _P],
    "cuca_sum_norm_shift_supported": [_I],
    "cuca_sum_norm_shift": [_P, _P, _P, _P, _F, _F, _P, _P, _P, _P, _I, _P, _P, _P, _I, _I, _I, _P],
    "cuca_shift_rows": [_P, _P, _P, _P, _I, _P, _P, _P, _P, _I, _I, _I, _P],
    "cuca_moe_glu_capped_dense": [_P, _P, _I, _P, _I, _I, _I, _I, _I, _F, _F, _F, _P],
}

_lock = threading.Lock()
_lib = None


def load(verbose: bool = True):
    """Build (if needed) and load the library; cached after the first call."""
    global _lib
    if _lib is not None:
        return _lib
    with _lock:
        if _lib is not None:
            return _lib
        try:
            path = _build.build(verbose=verbose)
        except _build.BuildError as e:
            raise KernelLibraryError(f"the CUDA kernel library of cuca_b200 could not be built: {e}") from e
        try:
            lib = ctypes.CDLL(str(path))
        except OSError as e:
            raise KernelLibraryError(f"the CUDA kernel library {path} could not be loaded: {e}") from e
        lib.cuca_last_error.restype = ctypes.c_char_p
        lib.cuca_last_error.argtypes = []
        for name, args in _SIGNATURES.items():
            try:
                fn = getattr(lib, name)
            except AttributeError as e:
                raise KernelLibraryError(f"{path} lacks `{name}`: stale build? remove {path.parent}") from e
            fn.restype = c_int
            fn.argtypes = args
        _lib = lib
        return lib


def declare(name: str, argtypes: list) -> None:
    """Declare a further exported function (used by kernels added later in this package)."""
    _SIGNATURES[name] = argtypes
    if _lib is not None:
        fn = getattr(_lib, name)
        fn.restype = c_int
        fn.argtypes = argtypes


launches = 0  # kernels launched through this library by this process (bench.py reports it)


def check(code: int, what: str) -> None:
    global launches
    launches += 1
    if code != 0:
        msg = _lib.cuca_last_error().decode(errors="replace") if _lib is not None else ""
        raise KernelError(f"{what}: {msg or 'error ' + str(code)}")
