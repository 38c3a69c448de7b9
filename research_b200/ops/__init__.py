"""Kernel entry points. Every op runs the sm_100a kernel on CUDA tensors and an fp32-faithful
PyTorch reference on CPU tensors (the oracle the GPU tests compare against)."""

from ._util import KernelStatusError, check_status, status_tensor
from .attention import (
    decode_num_splits,
    gather_kv,
    paged_decode,
    paged_decode_reference,
    paged_prefill,
    paged_prefill_reference,
)
from .elementwise import (
    clamped_glu,
    clamped_glu_reference,
    embedding,
    layernorm_reference,
    layernorm_residual,
    layernorm_rows,
    rmsnorm,
    rmsnorm_reference,
    rope_kv_append,
    rope_kv_append_reference,
    rope_table,
    ChosenExperts,
    StreamNorm,
    poly_norm,
    softcap,
    stream_embed,
    stream_norm,
    stream_sandwich,
    token_side,
    frequency_table,
    swiglu,
    swiglu_backward,
    swiglu_reference,
    transpose,
)
from .experts import ExpertsGeometry, ExpertsScratch, experts_forward, pack_experts
from .flash import (
    flash_attention,
    flash_attn_varlen,
    flash_attn_varlen_backward,
    flash_attn_varlen_reference,
    flash_latent_prefill,
    flash_latent_supported,
    flash_paged_prefill,
)
from . import gemm as gemm_mod
from .gemm import gemm, gemm_f32, gemm_fp8, lm_head_sample, lm_head_sample_workspace, gemm_reference, gemm_symmetric, quantize_fp8, interleave_gate_up, linear
from .latent import (
    LatentGeometry,
    head_gemm_absorb,
    head_gemm_expand,
    latent_append,
    latent_attention,
    latent_gather,
    latent_plan,
    latent_query,
    latent_units,
    latent_workspace,
)
from .keyvalue import KeyValueGeometry, kv_append, kv_attention, kv_workspace
from .grouped import GroupedCache, GroupedGeometry, grouped_append, grouped_attention
from .recurrent import ChunkTable, DeltaRule, ForgetMix, RecurrentGeometry, RecurrentState, TimeMix, delta_chunks, delta_rows, gated_norm, recurrent_chunks, recurrent_scan, tanh_parts, time_mix_chunks, time_mix_decode, token_shift
from .sampling import sample_with_logprobs, sample_with_logprobs_reference, token_logprobs

def set_pdl(on: bool) -> None:
    """Enable programmatic dependent launch for the decode-path kernels (GEMM, norms, RoPE,
    attention, SwiGLU, embedding, sampling): consecutive kernels overlap prologue and tail."""
    from .. import _native

    for lib, fn in (("rb_gemm", "rb_gemm_set_pdl"), ("rb_ops", "rb_ops_set_pdl"), ("rb_attn", "rb_attn_set_pdl"),
                    ("rb_latent", "rb_latent_set_pdl"), ("rb_gemm_f32", "rb_gemm_f32_set_pdl"),
                    ("rb_recurrent", "rb_recurrent_set_pdl"), ("rb_moe", "rb_moe_set_pdl")):
        if _native.available(lib):      # a partial build has only the libraries its models need
            getattr(_native.load(lib), fn)(int(on))


__all__ = [
    "KernelStatusError", "check_status", "status_tensor", "decode_num_splits", "gather_kv", "paged_decode",
    "paged_decode_reference", "paged_prefill", "paged_prefill_reference", "embedding", "rmsnorm",
    "rmsnorm_reference", "rope_kv_append", "rope_kv_append_reference", "rope_table", "swiglu", "swiglu_backward",
    "swiglu_reference", "transpose", "gemm", "gemm_reference", "linear", "sample_with_logprobs",
    "sample_with_logprobs_reference", "token_logprobs", "set_pdl", "interleave_gate_up", "gemm_mod", "gemm_symmetric", "gemm_fp8", "quantize_fp8", "lm_head_sample", "lm_head_sample_workspace", "flash_attention", "flash_attn_varlen",
    "flash_attn_varlen_backward", "flash_attn_varlen_reference", "flash_paged_prefill", "flash_latent_prefill", "flash_latent_supported", "clamped_glu", "clamped_glu_reference",
    "layernorm_reference", "layernorm_residual", "layernorm_rows", "softcap", "gemm_f32", "LatentGeometry",
    "head_gemm_absorb", "head_gemm_expand", "latent_append", "latent_attention", "latent_gather", "latent_plan", "latent_query", "latent_units", "latent_workspace",
    "ExpertsGeometry", "ExpertsScratch", "experts_forward", "pack_experts", "KeyValueGeometry", "kv_append", "kv_attention", "kv_workspace",
    "ChunkTable", "RecurrentGeometry", "RecurrentState", "gated_norm", "recurrent_chunks", "recurrent_scan", "stream_embed", "stream_norm",
    "GroupedCache", "GroupedGeometry", "grouped_append", "grouped_attention", "TimeMix", "ForgetMix", "DeltaRule", "delta_chunks", "delta_rows", "ChosenExperts", "StreamNorm", "poly_norm", "stream_sandwich", "tanh_parts", "time_mix_chunks", "time_mix_decode", "token_shift", "token_side", "frequency_table",
]
