"""Argument types of the library's ``extern "C"`` entry points, one letter per argument:
``p`` pointer or stream, ``i`` int, ``l`` long long, ``f`` float, ``d`` double.  With these declared, the
callers pass plain Python numbers and addresses, which ctypes converts without a wrapper
object per argument (a prefill step makes about a hundred calls, and the host must keep ahead
of the GPU).  ``tests/test_signatures.py`` derives the same table from the CUDA sources."""
from __future__ import annotations

import ctypes

SIGNATURES = {
    "nb_attention_decode_supported": "iiiii",
    "nb_attention_decode_scratch": "iiiiippp",
    "nb_attention_decode": "piiipppppiiiiipiifiiipppiiip",
    "nb_attention_decode_static": "piiipppppiiiiipiifiiip",
    "nb_attention_decode_capped": "piiipppppiiiiipiiffpiiipiiiipppp",
    "nb_attention_decode_cluster_merge": "i",
    "nb_attention_decode_cluster_limit": "",
    "nb_attention_generic": "piiipppppiiiiipiifiip",
    "nb_attention_prefill_supported": "iiiiiii",
    "nb_attention_prefill_f32_supported": "iiii",
    "nb_attention_prefill_f32": "piiippppppiiiiipiifiiip",
    "nb_attention_prefill": "piiippppppiiiiipiifiiip",
    "nb_attention_prefill_tc_supported": "iiiiiiiii",
    "nb_attention_prefill_tc_error": "",
    "nb_attention_prefill_tc_set_wait_budget": "l",
    "nb_attention_prefill_tc": "piiiipppppipiiiiipiifiiiiippiiip",
    "nb_attention_prefill_tc_capped": "piiiipppppipiiiiipiiffpiiiiippiiip",
    "nb_attention_prefill_tc_masked": "piiiipppppipiiiiipiiffpiiipiiiiiippiiip",
    "nb_attention_prefill_tc_record": "i",
    "nb_gemm_simt": "pipipppiiiiip",
    "nb_gemm_skinny": "pippfpipppiiiiip",
    "nb_gemm_stream": "pippfppppiiiiip",
    "nb_gemm_stream_supported": "iiii",
    "nb_gemm_stream_plan": "iiiip",
    "nb_gemm_stream_tune": "i",
    "nb_gemm_stream_set_wait_budget": "l",
    "nb_gemm_skinny_norm_supported": "iii",
    "nb_gemm_tc_rows_supported": "iii",
    "nb_gemm_tc_rows_preferred": "iii",
    "nb_gemm_tc_rows_plan": "iiip",
    "nb_gemm_tc_rows_force_split": "i",
    "nb_gemm_tc_rows_set_wait_budget": "l",
    "nb_gemm_tc_rows": "pppppiiiiip",
    "nb_gemm_tcgen05_supported": "iiiii",
    "nb_gemm_tcgen05_error": "",
    "nb_gemm_tcgen05_set_wait_budget": "l",
    "nb_wait_probe": "pp",
    "nb_device_errors": "i",
    "nb_gemm_tcgen05_use_pairs": "i",
    "nb_gemm_tcgen05_tune": "ii",
    "nb_gemm_tcgen05": "pppppiiiiip",
    "nb_abi_version": "",
    "nb_set_overlap": "i",
    "nb_get_overlap": "",
    "nb_embed_pos": "ppppipiifp",
    "nb_embed_hashed": "ppppippipipiifiiip",
    "nb_ln_add": "ppfppfppiiip",
    "nb_rms_add": "ppfppfppiiip",
    "nb_act_rows": "piiippiiip",
    "nb_gather_mul": "ppippiiip",
    "nb_qk_norm_rope_append": "piiippfpifpppippipiiiiiiip",
    "nb_qkv_norm_rope_append": "piiiippfpifpppippipipiiiiiiiip",
    "nb_pool_blocks": "pppppipppiiiiiiip",
    "nb_attention_pooled_mma": "piippppppipppiiiiippiifiiiip",
    "nb_attention_prefill_masked": "piippppppiiiiippiiffiiipiiiip",
    "nb_attention_pooled": "pipppppipppiiiiiippifiiip",
    "nb_conv_rope_append": "piipipippppipippippiiiiiiiiiip",
    "nb_conv_act": "piippiipippippiiiip",
    "nb_conv_state_update": "piiipippiip",
    "nb_attention_capped": "pippppippiiiiiiippiffip",
    "nb_attention_masked": "pippppippiiiiiiippiffiiipiiip",
    "nb_selective_scan_supported": "i",
    "nb_selective_scan": "ppiiipppppiipippiipiip",
    "nb_linear_attention_supported": "ii",
    "nb_linear_attention": "piiiiippippiiipip",
    "nb_glu_rows": "piiiifpiiip",
    "nb_cast_cols": "ppiiiiip",
    "nb_rmsnorm_gated": "pppiipiiifp",
    "nb_rms_pair_add": "ppppffppfpiiip",
    "nb_delta_rule_supported": "i",
    "nb_delta_rule": "piiiiiipppfffppppppiiiiip",
    "nb_layernorm": "pppppiiifp",
    "nb_rmsnorm": "piipppiiifp",
    "nb_latent_append": "piipfpppipiiiip",
    "nb_latent_rope_append": "piipfpiifpiipiipppipiiiiip",
    "nb_head_linear": "piiipipiiipiiipiiiip",
    "nb_attention_latent": "piiipppipiiiiippiifiip",
    "nb_attention_latent_mma_supported": "iiii",
    "nb_attention_latent_mma": "pppppppiiiiippfiiiiippp",
    "nb_streams": "piiippppppppfpiiip",
    "nb_softcap_rows": "pflp",
    "nb_attention_differential": "pippppippiiiiiiipififffip",
    "nb_attention_differential_mma_supported": "iiiii",
    "nb_attention_differential_mma": "pipppppippiiiiiipfifffiip",
    "nb_attention_decode_maps_supported": "iiiii",
    "nb_attention_decode_maps": "pipppppiiiiipififffiipppp",
    "nb_moe_gemm_mma_supported": "iiii",
    "nb_moe_gemm_mma": "pipipiipppiiiiifp",
    "nb_head_linear_mma_supported": "iiiiii",
    "nb_head_linear_mma": "piiippiipiiipiiiip",
    "nb_moe_gemm_tc_set_wait_budget": "l",
    "nb_moe_gemm_tc_supported": "iiiiii",
    "nb_moe_gather": "pipipipiip",
    "nb_moe_gemm_tc": "pipiipppiiiiifp",
    "nb_moe_route": "piipiiiippp",
    "nb_moe_route_sigmoid": "piippiiiiiiiffppp",
    "nb_moe_group": "piipppp",
    "nb_moe_gemm_tiles": "ii",
    "nb_moe_gemm": "piipipiippipiiiiifp",
    "nb_moe_combine": "pippipip",
    "nb_kv_append": "piiiipppppiiiiip",
    "nb_advance_decode": "ppppip",
    "nb_repetition_penalty": "piipipfp",
    "nb_history_append": "pipppip",
    "nb_top_candidates": "piiiidppppp",
    "nb_argmax_split": "piipppip",
    "nb_argmax": "piipp",
    "nb_sample_temperature": "piifppp",
    "nb_sample_top_k": "piiifppp",
    "nb_sample_top_p": "piiiffppp",
    "nb_sample_top_p_max_k": "",
}

_CTYPE = {"p": ctypes.c_void_p, "i": ctypes.c_int, "f": ctypes.c_float, "d": ctypes.c_double,
          "l": ctypes.c_longlong}


def declare(lib) -> None:
    """Set ``argtypes`` (and ``int`` results) on every entry point of the loaded library."""
    for name, letters in SIGNATURES.items():
        fn = getattr(lib, name)
        fn.argtypes = [_CTYPE[c] for c in letters]
        fn.restype = ctypes.c_int
    lib.nb_set_overlap.restype = None
    lib.nb_attention_decode_scratch.restype = None
    lib.nb_last_error.argtypes = []
    lib.nb_last_error.restype = ctypes.c_char_p
    lib.nb_attention_decode_static_capacity.argtypes = []
    lib.nb_attention_decode_static_capacity.restype = ctypes.c_longlong
