"""ctypes signatures of the CUDA kernel library (``libipex_llm_cuda.so``).

Every launcher returns a ``cudaError_t`` (0 = success); ``check`` turns a failure into a Python exception.
"""
from __future__ import annotations

import ctypes

vp = ctypes.c_void_p
ci = ctypes.c_int
i64 = ctypes.c_int64
cf = ctypes.c_float

DT_F16, DT_BF16, DT_F32 = 0, 1, 2
WF_SYM_INT4, WF_ASYM_INT4, WF_LUT4, WF_FP8_E4M3, WF_FP8_E5M2, WF_INT8, WF_F16, WF_BF16 = range(8)

_SIGS = {
    "ipex_gemv_lowbit": [vp, ci, vp, vp, ci, ci, ci, ci, ci, vp, cf, cf, vp, vp, ci, ci, vp, ci, ci, vp],
    "ipex_gemv_lowbit_tma": [vp, ci, vp, vp, ci, ci, ci, ci, ci, vp, cf, cf, vp, vp, ci, ci, vp, ci, ci, vp, vp],
    "ipex_gemv_lowbit_stream": [vp, ci, vp, vp, ci, ci, ci, ci, ci, vp, cf, cf, vp, vp, ci, ci, vp, ci, ci, vp, vp],
    "ipex_gemv_lowbit_tma_ar": [vp, ci, vp, vp, ci, ci, ci, ci, ci, vp, cf, cf, vp, vp, ci, vp, ci, ci, vp, vp,
                                ci, ci, ci, vp, vp],
    "ipex_allreduce_oneshot": [vp, vp, vp, i64, ci, ci, ci, vp, ci, ci, vp],
    "ipex_allreduce_oneshot_epi": [vp, vp, vp, i64, ci, ci, ci, vp, ci, ci, vp, vp, ci, vp],
    "ipex_symm_barrier": [vp, ci, ci, vp, vp],
    "ipex_wait_timeout_probe": [vp, ci, ci, vp, vp],
    "ipex_rms_norm": [vp, vp, vp, vp, vp, i64, ci, cf, cf, ci, ci, vp],
    "ipex_layer_norm": [vp, vp, vp, vp, i64, ci, cf, ci, vp],
    "ipex_act_mul": [vp, vp, vp, i64, ci, ci, ci, vp],
    "ipex_softmax_inplace": [vp, i64, ci, ci, vp],
    "ipex_attn_prefill_tcgen05": [vp, vp, vp, vp, ci, ci, ci, ci, ci, i64, i64, i64, i64, cf, ci, ci, vp, vp],
    "ipex_attn_transpose_v": [vp, vp, ci, ci, ci, ci, i64, i64, ci, vp],
    "ipex_rwkv_wkv_v4": [vp, vp, vp, vp, vp, vp, vp, vp, ci, ci, ci, ci, vp],
    "ipex_rwkv_linear_attention_v5": [vp, vp, vp, vp, vp, vp, vp, ci, ci, ci, ci, vp],
    "ipex_rwkv_time_shift": [vp, vp, vp, vp, ci, ci, ci, ci, ci, vp],
    "ipex_rope_inplace": [vp, vp, vp, vp, ci, ci, ci, ci, ci, i64, i64, i64, i64, i64, i64, i64, i64, ci, ci, ci, vp],
    "ipex_kv_quant_e5m2": [vp, vp, i64, ci, i64, ci, vp],
    "ipex_kv_dequant_e5m2": [vp, vp, i64, ci, i64, ci, vp],
    "ipex_repetition_penalty": [vp, vp, ci, ci, ci, cf, ci, vp],
    "ipex_embedding": [vp, vp, vp, i64, ci, cf, ci, ci, vp],
    "ipex_argmax": [vp, vp, ci, ci, i64, ci, ci, vp],
    "ipex_attn_decode": [vp, vp, vp, vp, vp, vp, vp, ci, vp, vp, vp, vp, vp, ci, ci, ci, ci, ci, ci, ci, ci, ci, ci,
                         cf, cf, ci, ci, ci, vp],
    "ipex_quantize_to_tiles": [vp, vp, i64, i64, i64, ci, ci, ci, vp],
    "ipex_dequantize_tiles": [vp, vp, i64, i64, i64, ci, vp, ci, vp],
    "ipex_dequantize_blocks": [vp, vp, i64, ci, ci, ci, ci, vp],
    "ipex_dequantize_rows": [vp, vp, vp, i64, ci, ci, ci, ci, ci, vp],
}

_I64_RET = {
    "ipex_attn_decode_scratch_floats": [ci, ci, ci, ci, ci, ci],
    "ipex_attn_decode_counter_ints": [ci, ci, ci, ci],
}

# optional entry points: declared when the library exports them (kernels added over time)
_OPTIONAL = {
    "ipex_gemm_tcgen05": [vp, vp, vp, vp, vp, ci, ci, ci, i64, i64, i64, i64, ci, vp, vp],
    "ipex_gemm_tcgen05_token_tile": [ci],
    "ipex_gemm_lowbit_tcgen05": [vp, vp, vp, vp, vp, vp, ci, ci, ci, i64, i64, i64, ci, ci, ci, vp, vp],
    "ipex_gemm_lowbit_tcgen05_grouped": [vp, vp, vp, vp, vp, ci, ci, ci, ci, i64, i64, ci, ci, ci, ci, vp, vp],
    "ipex_lora_rs_adamw": [vp, vp, vp, vp, vp, vp, vp, vp, i64, ci, ci, cf, cf, cf, cf, cf, ci, ci, ci, vp, vp],
    "ipex_moe_softmax_topk": [vp, vp, vp, vp, ci, ci, ci, ci, ci, vp],
}


# the components of the decoders with a 32-bit residual stream (see native/build.py)
COMPONENT_SIGS = {
    "stream": {
        "ipex_argmax": _SIGS["ipex_argmax"],
        "ipex_gemv_rows_max": [ci, ci],
        "ipex_gemv_rows": [vp, i64, vp, i64, vp, cf, vp, vp, i64, vp, ci, vp, i64, ci, ci, ci, ci, ci, ci, cf, ci, ci, cf, cf,
                           vp, i64, i64, vp, ci, ci, vp],
        "ipex_moe_router_sigmoid": [vp, i64, vp, cf, vp, vp, vp, ci, ci, ci, ci, ci, ci, vp],
        "ipex_moe_router_softmax": [vp, i64, vp, vp, vp, ci, ci, ci, ci, ci, ci, ci, cf, ci, ci, vp],
        "ipex_moe_glu_rows": [vp, i64, vp, cf, vp, vp, vp, i64, vp, vp, ci, ci, ci, ci, ci, ci, ci, cf, cf, cf, ci, ci,
                              ci, ci, vp],
        "ipex_moe_down_rows": [vp, i64, vp, vp, vp, vp, i64, vp, ci, ci, ci, ci, ci, ci, ci, ci, ci, vp],
        "ipex_embed_stream": [vp, vp, vp, vp, vp, i64, vp, vp, vp, ci, ci, i64, cf, i64, i64, i64, ci, ci, ci, vp],
        "ipex_norm_stream": [vp, i64, vp, ci, vp, i64, vp, ci, ci, cf, ci, ci, vp],
        "ipex_add_norm_stream": [vp, i64, vp, i64, vp, vp, vp, i64, ci, ci, cf, ci, ci, vp],
        "ipex_add_sides": [vp, i64, vp, vp, vp, vp, i64, vp, vp, i64, ci, ci, cf, ci, ci, vp],
        "ipex_act_rows": [vp, i64, ci, ci, ci, ci, ci, vp, i64, i64, vp, ci, vp],
        "ipex_bias_rows": [vp, i64, ci, vp, ci, ci, ci, vp],
        "ipex_hyper_joint": [vp, vp, i64, vp, vp, vp, vp, vp, i64, ci, ci, ci, cf, ci, ci, vp],
        "ipex_glu_rows": [vp, i64, ci, vp, vp, i64, ci, ci, ci, ci, cf, cf, ci, vp],
        "ipex_softcap_f32": [vp, i64, cf, vp],
        "ipex_add_stream": [vp, vp, i64, ci, vp],
        "ipex_relu2_inplace": [vp, i64, ci, vp],
        "ipex_moe_sigmoid_topk": [vp, i64, vp, vp, ci, ci, ci, vp],
        "ipex_moe_softmax_grouped_topk": [vp, i64, vp, vp, vp, ci, vp, ci, ci, ci, ci, ci, ci, cf, ci, vp],
        "ipex_moe_group_slots": [vp, ci, ci, vp, vp, vp, vp],
        "ipex_moe_gather_slots": [vp, vp, vp, vp, vp, ci, ci, ci, ci, vp],
        "ipex_moe_glu_from_gu": [vp, vp, vp, ci, ci, cf, cf, ci, ci, vp],
        "ipex_moe_combine_slots": [vp, vp, vp, ci, ci, ci, ci, vp],
        "ipex_moe_combine_weighted": [vp, vp, vp, vp, vp, ci, ci, ci, ci, ci, vp],
        "ipex_gemm_plain": [vp, vp, vp, vp, ci, ci, ci, ci, ci, ci, vp],
        "ipex_gemm_stream": [vp, i64, vp, i64, vp, i64, vp, vp, ci, vp, i64, vp, vp, ci, ci, ci, ci, ci, ci, cf, cf,
                             ci, vp, i64, i64, vp, ci, ci, vp, vp],
        "ipex_packed_prefill_ok": [ci, ci, ci, ci, ci],
        "ipex_packed_prefill": [vp, i64, vp, i64, vp, i64, vp, i64, vp, i64, vp, vp, ci, ci, ci, ci, ci, ci, ci, ci,
                                ci, ci, ci, vp, vp, i64, cf, ci, vp, i64, vp, i64, vp, ci, cf, ci, vp, vp],
    },
    "latent": {
        "ipex_latent_prep": [vp, i64, vp, i64, vp, cf, vp, vp, vp, vp, vp, vp, vp, i64, i64, vp, ci, ci, ci, ci, ci, ci,
                             ci, ci, vp],
        "ipex_latent_prompt_prep": [vp, i64, vp, i64, vp, cf, vp, vp, vp, vp, vp, vp, i64, i64, vp, i64, vp, i64, ci,
                                    ci, ci, ci, ci, ci, ci, ci, vp],
        "ipex_latent_row": [ci, ci, ci],
        "ipex_latent_attn_fast": [ci, ci, ci],
        "ipex_latent_attn": [vp, vp, i64, vp, i64, i64, vp, vp, vp, vp, vp, ci, ci, ci, ci, ci, ci, ci, cf, ci, ci, ci,
                             vp],
        "ipex_latent_uv": [vp, vp, vp, vp, i64, vp, i64, ci, ci, ci, ci, ci, ci, ci, vp],
    },
    "attention": {
        "ipex_kv_append": [vp, vp, i64, vp, i64, cf, vp, i64, i64, vp, i64, i64, vp, i64, vp, vp, ci, ci, ci, ci, ci,
                           ci, vp],
        "ipex_kv_pool": [vp, i64, i64, vp, i64, i64, vp, i64, i64, vp, i64, i64, vp, i64, vp, i64, vp, vp, vp, vp, vp, vp, ci, ci,
                         ci, ci, ci, ci, ci, vp],
        "ipex_qk_prepare": [vp, i64, vp, vp, vp, vp, vp, ci, ci, cf, vp, vp, ci, ci, ci, ci, ci, ci, vp],
        "ipex_kv_attn": [vp, vp, vp, i64, vp, i64, cf, vp, i64, i64, vp, i64, i64, vp, i64, vp, vp, vp, ci, ci, ci, ci,
                         ci, ci, ci, ci, vp, vp, i64, cf, ci, ci, vp, vp, ci, ci, cf, vp, vp, ci, vp, i64, i64, vp, i64, i64, ci,
                         cf, ci, ci, vp],
    },
    "recurrent": {
        "ipex_ring_tail": [vp, i64, vp, vp, vp, vp, vp, ci, ci, ci, ci, vp],
        "ipex_gated_norm": [vp, vp, i64, vp, ci, ci, vp, i64, ci, ci, ci, cf, cf, ci, vp],
        "ipex_gated_group_norm": [vp, vp, i64, vp, vp, i64, ci, ci, ci, cf, ci, ci, vp],
    },
    "delta": {
        "ipex_delta_chunks_ok": [ci, ci],
        "ipex_delta_fused_ok": [ci],
        "ipex_delta_step": [vp, i64, ci, vp, vp, vp, vp, vp, vp, vp, vp, vp, vp, vp, ci, vp, cf, vp, i64, vp, ci, ci,
                            ci, ci, ci, ci, ci, vp],
        "ipex_delta_chunks": [vp, i64, vp, vp, vp, vp, vp, vp, vp, vp, vp, vp, vp, ci, vp, vp, ci, ci, vp, vp, ci, ci,
                              ci, ci, ci, ci, vp, vp],
    },
    "general_delta": {
        "ipex_general_chunks_ok": [ci, ci, ci, cf],
        "ipex_general_fused_ok": [ci],
        "ipex_general_step": [vp, i64, ci, vp, i64, vp, vp, vp, vp, vp, vp, vp, vp, vp, ci, vp, cf, vp, i64, vp, ci, ci, ci, ci,
                              cf, ci, ci, vp],
        "ipex_general_chunks": [vp, i64, vp, i64, vp, vp, vp, vp, vp, vp, vp, vp, vp, ci, vp, vp, ci, ci, vp, vp, ci, ci, ci,
                                ci, cf, ci, vp, vp],
    },
    "ssd": {
        "ipex_ssd_chunks_ok": [ci, ci, ci],
        "ipex_ssd_step": [vp, i64, vp, i64, vp, vp, vp, vp, vp, vp, vp, vp, vp, vp, vp, vp, ci, vp, ci, ci, ci, ci, ci, ci, ci,
                          vp],
        "ipex_ssd_chunks": [vp, i64, vp, i64, vp, vp, vp, vp, vp, vp, vp, vp, vp, vp, vp, vp, ci, vp, vp, ci, ci, vp, vp, vp,
                            ci, ci, ci, ci, ci, ci, vp, vp],
    },
    "linear": {
        "ipex_linear_chunks_ok": [ci, ci, ci],
        "ipex_linear_fused_ok": [ci],
        "ipex_linear_step": [vp, i64, ci, vp, vp, vp, vp, vp, vp, vp, vp, vp, ci, vp, cf, cf, vp, i64, vp, ci, ci, ci, ci,
                             cf, ci, ci, vp],
        "ipex_linear_chunks": [vp, i64, vp, vp, vp, vp, vp, vp, vp, vp, vp, ci, vp, vp, ci, ci, vp, vp, ci, ci, ci, ci,
                               cf, ci, vp, vp],
    },
}


# scratch sizes of the chunked recurrences: (dim, vdim) -> floats
_SCRATCH_FLOATS = {"delta": ("ipex_delta_scratch_floats",), "general_delta": ("ipex_general_scratch_floats",),
                   "linear": ("ipex_linear_scratch_floats",), "ssd": ("ipex_ssd_group_floats", "ipex_ssd_head_floats")}


def declare_component(lib: ctypes.CDLL, name: str):
    for fn_name, args in COMPONENT_SIGS[name].items():
        fn = getattr(lib, fn_name)
        fn.argtypes, fn.restype = args, ci
    if name == "stream":
        lib.ipex_gemv_rows_tune.argtypes, lib.ipex_gemv_rows_tune.restype = [ci], None
    for fn_name in _SCRATCH_FLOATS.get(name, ()):
        fn = getattr(lib, fn_name)
        fn.argtypes, fn.restype = [ci, ci], i64


def declare(lib: ctypes.CDLL):
    for name, args in _SIGS.items():
        fn = getattr(lib, name)
        fn.argtypes = args
        fn.restype = ci
    for name, args in _I64_RET.items():
        fn = getattr(lib, name)
        fn.argtypes = args
        fn.restype = i64
    lib.ipex_gemv_tma_tune.argtypes = [ci, ci, ci]
    lib.ipex_gemv_tma_tune.restype = None
    for name, args in _OPTIONAL.items():
        fn = getattr(lib, name, None)
        if fn is not None:
            fn.argtypes = args
            fn.restype = ci


_CUDA_ERRORS = {1: "invalid value", 2: "out of memory", 98: "invalid device function", 700: "illegal address",
                701: "launch out of resources", 715: "illegal instruction", 719: "launch failure"}


def check(code: int, what: str):
    if code != 0:
        raise RuntimeError(f"ipex_llm_b200 CUDA kernel '{what}' failed: cudaError {code} "
                           f"({_CUDA_ERRORS.get(code, 'see cuda_runtime_api.h')})")


def dtype_code(torch_dtype) -> int:
    import torch
    if torch_dtype == torch.float16:
        return DT_F16
    if torch_dtype == torch.bfloat16:
        return DT_BF16
    if torch_dtype == torch.float32:
        return DT_F32
    raise TypeError(f"unsupported activation dtype {torch_dtype}")
