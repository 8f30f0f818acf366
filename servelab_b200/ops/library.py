"""Loads the compiled kernel libraries and declares their C signatures.

The kernels are the only implementation of their operations: there is no CPU or
framework fallback.  If the library cannot be built or loaded, or no CUDA device
is present, the first use raises ``KernelsUnavailable``.
"""

from __future__ import annotations

import ctypes
from ctypes import c_float, c_int, c_longlong, c_void_p
from typing import Dict

from ..csrc import build as _build


class KernelsUnavailable(RuntimeError):
    pass


class KernelError(RuntimeError):
    pass


P, I, F, LL = c_void_p, c_int, c_float, c_longlong

_CORE_SIGNATURES = {
    "slb_embedding_f32": [P, P, P, I, I, I, F, P],
    "slb_embedding_bf16": [P, P, P, I, I, I, F, P],
    "slb_logit_transform": [P, I, I, I, F, F, P],
    "slb_add_rmsnorm_f32": [P, P, P, P, P, I, I, F, P],
    "slb_add_rmsnorm_bf16": [P, P, P, P, P, I, I, F, P],
    "slb_swiglu_f32": [P, P, I, I, I, I, I, P],
    "slb_swiglu_bf16": [P, P, I, I, I, I, I, P],
    "slb_qkv_rope_cache_f32": [P, I, P, P, P, P, I, I, I, P, I, P, I, P, P, I, I, I, I, P],
    "slb_qkv_rope_cache_bf16": [P, I, P, P, P, P, I, I, I, P, I, P, I, P, P, I, I, I, I, P],
    "slb_cache_write_status": [I],
    "slb_paged_attention_generic_f32": [P, I, P, P, P, I, P, I, P, P, P, P, I, I, I, I, I, I, F, I, P, P, P, P],
    "slb_paged_attention_generic_bf16": [P, I, P, P, P, I, P, I, P, P, P, P, I, I, I, I, I, I, F, I, P, P, P, P],
    "slb_mix_heads_gate_f32": [P, P, I, I, P, I, P, P, I, P, I, I, I, I, I, P],
    "slb_mix_heads_gate_bf16": [P, P, I, I, P, I, P, P, I, P, I, I, I, I, I, P],
    "slb_dyt_add_norm_f32": [P, I, P, I, P, P, P, P, P, P, P, I, P, I, I, P],
    "slb_dyt_add_norm_bf16": [P, I, P, I, P, P, P, P, P, P, P, I, P, I, I, P],
    "slb_qk_conv_cache_f32": [P, I, P, I, P, P, P, P, P, P, I, I, I, F, I, P, I, P, I, I, I, I, I, I, LL, P],
    "slb_qk_conv_cache_bf16": [P, I, P, I, P, P, P, P, P, P, I, I, I, F, I, P, I, P, I, I, I, I, I, I, LL, P],
    "slb_conv_cache_status": [I],
    "slb_paged_attention_generic_status": [I],
    "slb_paged_attention_generic_tile_rows": [],
    "slb_gemm_simt_f32": [P, I, P, I, P, I, P, I, I, I, P],
    "slb_gemm_simt_bf16": [P, I, P, I, P, I, P, I, I, I, P],
    "slb_gemm_simt_bf16_f32out": [P, I, P, I, P, I, P, I, I, I, P],
    "slb_sample_rows": [P, I, I, I, P, P, P, P, P, P, P, P],
    "slb_gemm_tc_decode_bf16": [P, I, P, I, P, I, P, P, I, I, I, I, I, I, I, I, P, I, F, I, P],
    "slb_split_sum": [P, P, I, P, I, I, I, I, P],
    "slb_gemm_tc_cluster_bf16": [P, I, P, I, P, I, P, I, I, I, I, I, P, I, F, I, P],
    "slb_gemm_tc_qkv_rope_bf16": [P, I, P, I, P, P, P, P, I, I, I, P, I, P, I, P, P, I, I, I, I, I, I, I,
                                  P, I, F, I, P],
    "slb_gemm_tc_resid_norm_bf16": [P, I, P, I, P, P, I, P, P, I, P, I, I, I, I, I, I, P],
    "slb_gemm_tc_resid_dyt_bf16": [P, I, P, I, P, I, P, P, P, P, P, P, P, I, I, I, I, I, I, I, P],
    "slb_add_rmsnorm_parts_bf16": [P, P, I, LL, P, P, P, P, I, I, F, P],
    "slb_qkv_rope_cache_parts_bf16": [P, I, LL, I, P, P, P, P, I, I, I, P, I, P, I, P, P, I, I, I, I, P],
    "slb_gemm_tc_status": [I],
    "slb_ln_add_norm_f32": [P, I, P, I, P, P, F, P, P, F, P, I, P, I, I, P],
    "slb_ln_add_norm_bf16": [P, I, P, I, P, P, F, P, P, F, P, I, P, I, I, P],
    "slb_head_prep_f32": [P, I, P],
    "slb_head_prep_bf16": [P, I, P],
    "slb_head_prep_status": [I],
    "slb_sigmoid_gate_f32": [P, I, P, I, P, I, I, I, I, P],
    "slb_sigmoid_gate_bf16": [P, I, P, I, P, I, I, I, I, P],
    "slb_attention_kv_tile_rows": [],
    "slb_attention_kv_status": [I],
    "slb_attention_kv_f32": [P, I, P, P, I, P, I, P, I, P, P, P, P, I, I, I, I, I, I, I, F, I, P, I, F, P, I, P, P, F,
                             P],
    "slb_attention_kv_bf16": [P, I, P, P, I, P, I, P, I, P, P, P, P, I, I, I, I, I, I, I, F, I, P, I, F, P, I, P, P, F,
                              P],
    "slb_gemm_simt_batched_f32": [P, I, P, I, P, I, I, I, I, I, LL, LL, LL, P],
    "slb_gemm_simt_batched_bf16": [P, I, P, I, P, I, I, I, I, I, LL, LL, LL, P],
    "slb_gemm_simt_batched_bf16_f32out": [P, I, P, I, P, I, I, I, I, I, LL, LL, LL, P],
    "slb_gemm_simt_tanh_f32": [P, I, P, I, P, I, P, I, I, I, P],
    "slb_tanh_linear_bf16": [P, I, P, I, P, I, P, I, I, I, P],
    "slb_dyt_parallel_f32": [P, P],
    "slb_dyt_parallel_bf16": [P, P],
    "slb_stream_rows_f32": [P, P],
    "slb_stream_rows_bf16": [P, P],
    "slb_short_conv_f32": [P, I, P, I, P, P, P, P, P, P, I, I, I, I, I, LL, P, P, I, P],
    "slb_short_conv_bf16": [P, I, P, I, P, P, P, P, P, P, I, I, I, I, I, LL, P, P, I, P],
    "slb_token_mix_max": [],
    "slb_embed_bigram_f32": [P, P, P, P, P, LL, I, P, I, P, LL, LL, LL, P, P, I, I, I, P],
    "slb_embed_bigram_bf16": [P, P, P, P, P, LL, I, P, I, P, LL, LL, LL, P, P, I, I, I, P],
    "slb_token_mix_f32": [P, I, P, I, P, LL, I, P, P, P, P, I, I, P],
    "slb_token_mix_bf16": [P, I, P, I, P, LL, I, P, P, P, P, I, I, P],
    "slb_delta_rule_max_dim": [],
    "slb_delta_rule_fuses": [I, I],
    "slb_delta_rule_f32": [P, I, P],
    "slb_delta_rule_bf16": [P, I, P],
    "slb_delta_chunk_tokens": [],
    "slb_delta_chunk_work_floats": [I],
    "slb_delta_chunk_f32": [P, I, P],
    "slb_delta_chunk_bf16": [P, I, P],
    "slb_gated_recurrence_f32": [P, I, I, P],
    "slb_gated_recurrence_bf16": [P, I, I, P],
    "slb_moe_tile_rows": [],
    "slb_moe_route": [P, I, I, I, I, I, I, F, I, P, P, P],
    "slb_moe_route_scored": [P, I, I, I, I, I, I, F, I, I, P, I, F, P, P, P],
    "slb_gated_act_f32": [P, P, I, I, I, I, I, I, F, F, P, P],
    "slb_gated_act_bf16": [P, P, I, I, I, I, I, I, F, F, P, P],
    "slb_rms_norm_rows_f32": [P, I, P, F, P, I, I, I, P],
    "slb_rms_norm_rows_bf16": [P, I, P, F, P, I, I, I, P],
    "slb_norm_sum2_f32": [P, I, P, I, P, P, F, F, P, I, I, I, P],
    "slb_norm_sum2_bf16": [P, I, P, I, P, P, F, F, P, I, I, I, P],
    "slb_attention_kv_maps_f32": [P, I, P, I, I, P, I, P, I, P, I, P, P, P, P, I, I, I, I, I, I, I, F, I, P],
    "slb_attention_kv_maps_bf16": [P, I, P, I, I, P, I, P, I, P, I, P, P, P, P, I, I, I, I, I, I, I, F, I, P],
    "slb_hyper_max_streams": [],
    "slb_state_space_max_state": [],
    "slb_state_space_chunk_tokens": [],
    "slb_state_space_chunk_bf16": [P, I, P],
    "slb_embed_norm_streams_f32": [P, P, P, F, P, I, I, I, I, P],
    "slb_embed_norm_streams_bf16": [P, P, P, F, P, I, I, I, I, P],
    "slb_hyper_mix_norm_f32": [P, P, I, P, P, P, P, F, P, I, P, I, I, I, P],
    "slb_hyper_mix_norm_bf16": [P, P, I, P, P, P, P, F, P, I, P, I, I, I, P],
    "slb_gate_group_norm_f32": [P, I, P, I, I, P, F, F, P, I, I, I, I, P],
    "slb_post_add_rmsnorm_f32": [P, P, P, I, LL, P, P, F, P, P, P, I, I, F, P],
    "slb_state_space_f32": [P, I, P],
    "slb_group_norm_gate_f32": [P, I, I, P, P, F, F, P, I, I, P, I, I, I, I, P],
    "slb_gate_group_norm_bf16": [P, I, P, I, I, P, F, F, P, I, I, I, I, P],
    "slb_post_add_rmsnorm_bf16": [P, P, P, I, LL, P, P, F, P, P, P, I, I, F, P],
    "slb_state_space_bf16": [P, I, P],
    "slb_group_norm_gate_bf16": [P, I, I, P, P, F, F, P, I, I, P, I, I, I, I, P],
    "slb_decay_attention_max_dim": [],
    "slb_decay_attention_f32": [P, I, P],
    "slb_decay_attention_bf16": [P, I, P],
    "slb_decay_chunk_max_dim": [],
    "slb_decay_chunk_tokens": [],
    "slb_decay_chunk_bf16": [P, I, I, P],
    "slb_decay_gated_chunk_max_dim": [],
    "slb_decay_gated_chunk_tokens": [],
    "slb_decay_gated_chunk_f32": [P, I, P],
    "slb_decay_gated_chunk_bf16": [P, I, P],
    "slb_router_logits_f32": [P, I, P, I, P, I, I, I, I, P],
    "slb_router_logits_bf16": [P, I, P, I, P, I, I, I, I, P],
    "slb_moe_plan_ints": [I, I],
    "slb_moe_plan": [P, I, I, P, P],
    "slb_moe_gate_up_f32": [P, I, P, I, P, I, P, I, I, I, I, I, I, F, F, P, P],
    "slb_moe_gate_up_bf16": [P, I, P, I, P, I, P, I, I, I, I, I, I, F, F, P, P],
    "slb_moe_down_f32": [P, I, P, I, P, I, P, I, I, I, I, I, P],
    "slb_moe_down_bf16": [P, I, P, I, P, I, P, I, I, I, I, I, P],
    "slb_moe_gate_up_mma_bf16": [P, I, P, I, P, I, P, I, I, I, I, I, I, F, F, P, P],
    "slb_moe_down_mma_bf16": [P, I, P, I, P, I, P, I, I, I, I, I, P],
    "slb_moe_combine_f32": [P, I, P, P, I, P, I, I, I, I, P],
    "slb_moe_combine_bf16": [P, I, P, P, I, P, I, I, I, I, P],
    "slb_moe_combine_bf16_rows": [P, I, P, P, I, P, I, I, I, I, P],
}

# optional entry points: declared when the library exports them
_OPTIONAL_SIGNATURES = {}

_libs: Dict[str, ctypes.CDLL] = {}
_pdl = True
_pdl_early = False
trace_buffer = None        # device address of a timeline buffer (``ops.timeline``) or None


def loaded_libraries():
    return list(_libs.values())


def set_pdl(on: bool) -> None:
    """Programmatic dependent launch for every kernel of this package: a kernel may
    be scheduled while its predecessor in the stream drains (each kernel waits on
    the device for its predecessor before it touches activations).  Applies to the
    libraries loaded so far and to those loaded later."""
    global _pdl
    _pdl = bool(on)
    for lib in _libs.values():
        lib.slb_set_pdl(1 if _pdl else 0)


def pdl_enabled() -> bool:
    return _pdl


_FLAG_PDL_EARLY, _FLAG_EVICT_FIRST = 1, 2
_evict_first = True


def _kernel_flags() -> int:
    return (_FLAG_PDL_EARLY if _pdl_early else 0) | (_FLAG_EVICT_FIRST if _evict_first else 0)


def set_pdl_early(on: bool) -> None:
    """The long kernels (matrix products, decode attention) let their successor be scheduled
    at their start instead of after their main loop: its blocks become resident beside theirs
    wherever an SM has room and fetch their first weight tiles meanwhile."""
    global _pdl_early
    _pdl_early = bool(on)
    for lib in _libs.values():
        lib.slb_set_kernel_flags(_kernel_flags())


def set_evict_first(on: bool) -> None:
    """What a step streams once (weights, the cache) is fetched with the L2 policy "evict first",
    so that the activations between the kernels stay in the L2 cache (on by default)."""
    global _evict_first
    _evict_first = bool(on)
    for lib in _libs.values():
        lib.slb_set_kernel_flags(_kernel_flags())


def _apply_switches(lib: ctypes.CDLL) -> None:
    lib.slb_set_pdl.argtypes = [I]
    lib.slb_set_pdl(1 if _pdl else 0)
    lib.slb_set_kernel_flags.argtypes = [I]
    lib.slb_set_kernel_flags(_kernel_flags())
    lib.slb_set_trace.argtypes = [P, I]
    lib.slb_set_trace(trace_buffer, len(_libs))


def _declare(lib: ctypes.CDLL, sigs: dict, required: bool) -> None:
    for name, args in sigs.items():
        try:
            fn = getattr(lib, name)
        except AttributeError:
            if required:
                raise KernelsUnavailable(f"kernel library lacks symbol {name}") from None
            continue
        fn.argtypes = args
        fn.restype = c_int


def core() -> ctypes.CDLL:
    lib = _libs.get("core")
    if lib is None:
        try:
            path = _build.ensure_library()
            lib = ctypes.CDLL(path)
        except (OSError, _build.BuildError) as e:
            raise KernelsUnavailable(f"the servelab_b200 CUDA kernels are not available: {e}") from e
        _declare(lib, _CORE_SIGNATURES, True)
        _declare(lib, _OPTIONAL_SIGNATURES, False)
        _apply_switches(lib)
        _libs["core"] = lib
    return lib


_ATTN_SIGNATURES = {
    "slb_prefill_attention_bf16": [P, I, P, P, P, I, P, I, P, P, P, P, I, I, I, I, I, F, I, P],
    "slb_decode_attention_bf16": [P, I, P, P, P, I, P, I, P, P, I, I, I, I, I, F, I, I, P],
    "slb_prefill_attention_tile_rows": [],
    "slb_decode_attention_max_splits": [],
    "slb_attention_head_dim": [],
    "slb_attention_status": [I],
    "slb_prefill_attention_tc_supported": [I, I],
    "slb_prefill_attention_tc_tile_rows": [I],
    "slb_prefill_attention_tc_status": [I],
    "slb_prefill_attention_tc_where": [P],
    "slb_decode_attention_ws_bf16": [P, I, P, P, P, I, P, I, P, P, P, I, I, I, I, I, F, I, I, I, F, I, I, P],
    "slb_decode_attention_ws_max_cluster_splits": [],
    "slb_decode_attention_ws_supported": [I],
    "slb_decode_attention_ws_status": [I],
    "slb_decode_attention_ws_splits_used": [I],
    "slb_decode_attention_ws_max_splits": [],
    "slb_decode_attention_ws_tile_keys": [],
    "slb_talk_attention_value_heads": [],
    "slb_talk_prefill_attention_bf16": [P, I, P, P, P, I, P, P, P, P, I, I, I, I, I, F, I, P, P, P, I, P],
    "slb_talk_decode_attention_bf16": [P, I, P, P, P, I, P, I, I, I, I, I, F, I, I, P, P, P, P, I, P],
}


def attention(head_dim: int) -> ctypes.CDLL:
    key = f"attn{head_dim}"
    lib = _libs.get(key)
    if lib is None:
        try:
            lib = ctypes.CDLL(_build.attention_library(head_dim))
        except (OSError, _build.BuildError) as e:
            raise KernelsUnavailable(
                f"the attention kernels for head size {head_dim} are not available: {e}") from e
        _declare(lib, _ATTN_SIGNATURES, True)
        if hasattr(lib, "slb_prefill_attention_tc_bf16"):
            lib.slb_prefill_attention_tc_bf16.argtypes = [P, I, P, P, P, I, P, I, P, P, P, P, I, I, I, I, I,
                                                          F, I, P]
            lib.slb_prefill_attention_tc_bf16.restype = I
        lib.slb_decode_attention_scratch_bytes.argtypes = [I, I, I]
        lib.slb_decode_attention_scratch_bytes.restype = ctypes.c_longlong
        lib.slb_decode_attention_ws_scratch_bytes.argtypes = [I, I, I]
        lib.slb_decode_attention_ws_scratch_bytes.restype = ctypes.c_longlong
        lib.slb_decode_attention_ws_counters.argtypes = [I, I, I]
        lib.slb_decode_attention_ws_counters.restype = ctypes.c_longlong
        if lib.slb_attention_head_dim() != head_dim:
            raise KernelsUnavailable(f"attention library built for head size "
                                     f"{lib.slb_attention_head_dim()}, wanted {head_dim}")
        _apply_switches(lib)
        _libs[key] = lib
    return lib


_ATTN_KV_SIGNATURES = {
    "slb_attention_kv_mma_key_dim": [],
    "slb_attention_kv_mma_value_dim": [],
    "slb_attention_kv_mma_tile_rows": [],
    "slb_attention_kv_mma_status": [I],
    "slb_attention_kv_mma_bf16": [P, I, P, P, I, P, I, P, I, P, P, P, P, I, I, I, I, I, F, I, P, I, I, P, P, I, P],
    "slb_attention_kv_mma_capped_bf16": [P, I, P, P, I, P, I, P, I, P, P, P, P, I, I, I, I, I, F, I, P, I, I, P, P, I,
                                         F, P, I, P, P, F, P],
    "slb_attention_kv_mma_max_splits": [],
    "slb_attention_kv_mma_resident": [I, I],
    "slb_attention_kv_mma_maps_bf16": [P, I, P, P, I, P, I, P, I, P, P, P, P, I, I, I, I, I, F, I, I, P, P, I, P],
    "slb_attention_kv_mma_folded_bf16": [P, I, P, P, I, P, I, P, I, P, P, P, P, I, I, I, I, I, F, I, I, P, P, I, P],
    "slb_attention_kv_tc_supported": [I, I, I],
    "slb_attention_kv_tc_tile_rows": [I],
    "slb_attention_kv_tc_status": [I],
    "slb_attention_kv_tc_where": [P],
    "slb_attention_kv_tc_bf16": [P, I, P, P, I, P, I, P, I, P, P, P, P, I, I, I, I, I, F, I, P, I, P],
    "slb_attention_kv_tc_capped_bf16": [P, I, P, P, I, P, I, P, I, P, P, P, P, I, I, I, I, I, F, I, P, I, F, P, I, P,
                                        P, F, P],
    "slb_attention_kv_tc_maps_bf16": [P, I, P, P, P, I, P, I, P, P, P, P, I, I, I, I, I, I, F, I, P],
}


def attention_kv(key_dim: int, value_dim: int) -> ctypes.CDLL:
    """The tensor-core attention kernels for keys of ``key_dim`` and values of ``value_dim``."""
    key = f"attn_k{key_dim}v{value_dim}"
    lib = _libs.get(key)
    if lib is None:
        try:
            lib = ctypes.CDLL(_build.attention_kv_library(key_dim, value_dim))
        except (OSError, _build.BuildError) as e:
            raise KernelsUnavailable(f"the attention kernels for key size {key_dim} and value size "
                                     f"{value_dim} are not available: {e}") from e
        _declare(lib, _ATTN_KV_SIGNATURES, True)
        if (lib.slb_attention_kv_mma_key_dim(), lib.slb_attention_kv_mma_value_dim()) != (key_dim, value_dim):
            raise KernelsUnavailable("attention library built for other sizes than asked for")
        _apply_switches(lib)
        _libs[key] = lib
    return lib


# measurements: called with the kernel's name after every launch of this package's kernels
# (``ops.profile.StepProfile`` records a CUDA event there); None costs one comparison a launch
after_launch = None


def check(code: int, what: str) -> None:
    if code == 0:
        if after_launch is not None:
            after_launch(what)
        return
    if code == -1:
        raise KernelError(f"{what}: arguments refused (a size or pointer the kernel does not take)")
    if code == -2:
        raise KernelError(f"{what}: a size is beyond the kernel's stated maximum")
    raise KernelError(f"{what}: CUDA error {code} at launch")
