"""Loads the CUDA library and declares its C interface for ``ctypes``.

The engine has no path without this library: :func:`library` raises if it can
neither be found nor built.
"""

from __future__ import annotations

import ctypes
from ctypes import c_float, c_int, c_longlong, c_uint, c_ulonglong, c_void_p
from functools import lru_cache

from .build import BuildError, ensure_built

_P = c_void_p

# name -> argument types (every function returns a cudaError_t as int unless noted)
_SIGNATURES: dict[str, list] = {
    "tk_embed_gather": [_P, c_int, _P, _P, c_int, c_int, c_int, c_float, c_int, _P, _P],
    "tk_embed_bigram": [_P, _P, c_int, _P, _P, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int,
                        c_longlong, c_longlong, c_float, _P, _P],
    "tk_sum_rmsnorm": [_P] + 3 * [_P, c_int, c_int, c_longlong, _P, _P] + [_P, _P, _P, _P, _P, c_int, c_int, c_int, c_float,
                                                                          c_int, _P],
    "tk_step_begin": [_P, c_int, c_int, _P, c_int, _P, c_longlong, _P, _P, _P, _P, _P, c_int, c_int, _P, _P],
    "tk_decode_begin": [_P, c_int, c_int, _P, c_int, _P, c_longlong, _P, c_int, c_int, _P, _P, _P, _P, _P],
    "tk_sample_slots": [_P, c_longlong, _P, _P, c_int, _P, c_int, c_int, _P, _P],
    "tk_wait_probe": [c_uint, _P, _P],
    "tk_probe_mma_issue": [c_int, c_int, c_int, _P, _P, _P],
    "tk_probe_softmax_tile": [c_int, c_int, c_int, c_int, _P, _P],
    "tk_gemm_chain": [_P, c_int, c_int, _P, _P, _P, c_int, _P],
    "tk_gemm_chain_blocks": [],
    "tk_gemm_chain_max_phases": [],
    "tk_slot_words": [],
    "tk_add_rmsnorm": [_P, _P, _P, c_int, c_longlong, _P, _P, _P, c_int, c_int, c_float, c_int, _P],
    "tk_swiglu": [_P, _P, c_int, c_longlong, _P, c_int, c_int, c_int, c_int, c_int, _P],
    "tk_rope_kv": [_P, _P, c_int, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P,
                   c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                   c_float, c_int, _P],
    "tk_rope_table": [_P, _P, _P, c_int, c_int, c_float, _P],
    "tk_attention_plain": [_P, _P, _P, _P, _P, _P, _P, _P, _P, _P,
                           c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                           c_float, c_int, c_int, c_float, _P, c_int, c_longlong, c_longlong, c_int, c_int, c_int, _P,
                           _P, c_int, _P],
    "tk_latent_prepare": [_P, _P, c_int, c_longlong, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                          _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P,
                          c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_float, c_int, _P],
    "tk_attention_latent": [_P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, c_longlong, c_longlong,
                            c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_float, _P],
    "tk_attention_latent_takes": [c_int, c_int],
    "tk_heads_gate": [_P, _P, _P, c_int, c_longlong, c_int, c_int, _P, c_int, c_int, c_int, c_int, _P],
    "tk_delta_prepare": [_P, _P, c_int, c_longlong, c_int, c_int, c_int, c_int, c_int, c_int, _P, _P, _P, _P,
                         c_longlong, c_longlong, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P,
                         c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_float, c_float, c_int, c_int, c_int,
                         _P, _P, c_int, c_longlong, c_int, _P],
    "tk_low_rank": [_P, _P, c_int, c_longlong, c_int] + 2 * [c_int, c_int, _P, c_int, _P] + [c_int, c_int, _P],
    "tk_delta_scan": [_P, _P, _P, _P, _P, _P, c_longlong, _P, _P, _P, _P, _P,
                      c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P],
    "tk_delta_scan_cols": [c_int, c_int, c_int],
    "tk_gemm_f32_batched": [_P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_longlong, c_longlong,
                            c_longlong, _P],
    "tk_branch_norm_add": [_P, _P, _P, c_int, c_longlong, _P, _P, _P, _P, _P, c_int, c_int, c_float, c_float,
                           c_int, c_int, c_int, _P],
    "tk_branch_pair_norm_add": [_P] + 2 * [_P, _P, c_int, c_longlong, _P] + [_P, _P, _P, c_int, c_int, c_float, c_float, c_int,
                                                                             _P],
    "tk_short_conv": [_P, _P, c_int, c_longlong, _P, c_int, c_int, _P, _P, _P, _P, _P, _P, _P, _P, _P,
                      c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P],
    "tk_hgrn2_prepare": [_P, _P, c_int, c_longlong, c_int, c_int, c_int, c_int, _P, _P, _P, c_int, c_int, c_int, c_int,
                         c_int, _P],
    "tk_mlstm_prepare": [_P, _P, c_int, c_longlong, c_int, c_int, c_int, c_int, c_int, c_int, _P, _P, c_float, c_float,
                         _P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P],
    "tk_mlstm_out": [_P, _P, _P, _P, c_int, c_longlong, c_int, c_int, _P, _P, c_int, c_int, c_int, c_int, c_float,
                     c_float, c_int, _P],
    "tk_ssd_prepare": [_P, _P, _P, c_int, c_longlong, c_int, c_int, _P, _P, _P, c_int, c_int, c_int, c_int, c_int,
                       c_int, _P],
    "tk_ssd_out": [_P, _P, c_int, _P, _P, c_int, c_longlong, c_int, c_int, _P, _P, _P, c_int, c_int, c_int, c_int,
                   c_int, c_float, c_float, c_int, _P],
    "tk_gate_scale": [_P, _P, _P, c_int, c_longlong, c_int, c_int, _P, c_int, c_int, c_int, c_float, c_int, c_int, _P],
    "tk_retention_prepare": [_P, _P, c_int, c_longlong, c_int, c_int, c_int, c_int, _P, _P, c_int, c_int, c_float,
                             c_float, _P, c_int, c_int, c_int, c_int, c_int, _P],
    "tk_qkv_heads": [_P, _P, c_int, c_longlong, c_int, c_int, c_int, c_int, _P, _P, _P, _P, _P, c_int, c_float,
                     _P, c_int, c_int, c_float, c_int, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P,
                     c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P],
    "tk_map_difference": [_P, _P, c_longlong, c_int, c_int, c_int, c_int, c_float, c_float, c_float, c_int, _P],
    "tk_hyper_mix_norm": [_P, _P, _P, c_int, c_longlong, c_int, _P, _P, _P, _P, _P, _P, _P, _P,
                          c_int, c_int, c_int, c_int, c_float, c_float, c_int, _P],
    "tk_logits_scale_cap": [_P, c_longlong, c_float, c_float, _P],
    "tk_unary_act": [_P, _P, c_int, c_longlong, _P, c_longlong, c_int, c_int, _P],
    "tk_qkv_rownorm": [_P, _P, c_int, c_longlong, c_int, c_int, c_int, c_int, _P, _P, _P, _P, _P, _P, _P, _P,
                       _P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                       c_float, c_int, _P],
    "tk_moe_tile_rows": [],
    "tk_moe_pad_rows": [],
    "tk_moe_route": 11 * [_P] + 13 * [c_int] + [_P],
    "tk_moe_gather": [_P, c_longlong, _P, _P, c_int, c_int, c_int, _P],
    "tk_moe_combine_rows": [_P, _P, _P, _P, c_int, c_int, c_int, _P],
    "tk_moe_ffn": [_P, c_longlong, c_int, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P],
    "tk_moe_combine": [_P, _P, _P, c_int, c_int, c_int, _P],
    "tk_moe_small_max_pairs": [],
    "tk_moe_small": [_P, c_longlong, c_int, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P],
    "tk_qkv_pairs": [_P, _P, c_int, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P,
                     c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                     c_float, c_int, _P],
    "tk_gla_prepare": [_P, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P, _P, _P, c_int, c_int, c_int, c_int, c_int,
                       c_float, c_float, c_int, _P],
    "tk_gla_scan": [_P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P],
    "tk_gla_out": [_P, _P, _P, c_int, c_int, c_int, _P, _P, c_int, c_float, c_int, c_int, c_int, c_float, c_int, c_int, _P],
    "tk_attention_decode": [_P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P,
                            c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                            c_float, c_float, _P, c_int, _P, _P, c_int, _P],
    "tk_attention_decode_balanced": [_P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P,
                                     c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                                     c_float, c_float, _P, c_int, _P, _P, c_int, _P],
    "tk_attention_prefill": [_P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P,
                             c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                             c_float, _P],
    "tk_attention_prefill_tc": [_P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P,
                                c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                                c_float, c_float, _P, c_int, _P, _P, c_int, _P],
    "tk_attention_prefill_tc_takes": [c_int, c_int, c_int, c_int],
    "tk_attention_prefill_tc_rows": [],
    "tk_attention_prefill_tc_keys": [],
    "tk_attention_prefill_tc_record_ints": [],
    "tk_attention_prefill_tc_max_parts": [],
    "tk_gemm_bf16_tcgen05": [_P, _P, _P, _P, c_int, c_int, c_int, c_longlong, c_longlong,
                             c_int, c_int, c_int, c_int, c_int,
                             _P, c_int, c_float, c_float, _P, _P, _P, _P, _P],
    "tk_gemm_qkv_rope": [_P, _P, _P, c_int, c_int, c_longlong, c_longlong, c_int, c_int, c_int,
                         _P, c_int, c_float, c_float,
                         _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P,
                         c_int, c_int, c_int, c_int, c_int, c_int, c_float, _P],
    "tk_gemm_bf16_pair": [_P, _P, _P, _P, c_int, c_int, c_int, c_longlong, c_longlong, c_longlong, c_int, _P],
    "tk_gemm_bf16_pair_grouped": [_P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_longlong, c_longlong, c_longlong,
                                  c_int, _P],
    "tk_gemm_f32": [_P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P],
    "tk_sample": [_P, c_longlong, _P, _P, _P, _P, _P, _P, c_int, c_int, _P],
}


@lru_cache(maxsize=1)
def library() -> ctypes.CDLL:
    """The loaded library, compiled on first use if it is stale or absent."""
    try:
        path = ensure_built()
    except BuildError as exc:
        raise RuntimeError(
            f"tokamak_b200 needs its CUDA extension and could not build it: {exc}") from exc
    lib = ctypes.CDLL(str(path))
    for name, argtypes in _SIGNATURES.items():
        fn = getattr(lib, name)
        fn.argtypes = argtypes
        fn.restype = c_int
    for name, args in (("tk_gemm_chain_scratch_floats", [c_int]), ("tk_gemm_chain_counter_ints", [c_int]),
                       ("tk_attention_decode_balanced_scratch_floats", [c_int, c_int])):
        fn = getattr(lib, name)
        fn.argtypes = args
        fn.restype = c_longlong
    lib.tk_philox_u32.argtypes = [c_ulonglong, c_uint, ctypes.POINTER(c_uint)]
    lib.tk_philox_u32.restype = None
    return lib
