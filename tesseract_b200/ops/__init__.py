"""Functional ops. CUDA tensors are served by the native sm_100a kernels; CPU tensors by the torch
restatement of the reference's CPU math (which doubles as the test oracle)."""
from .attention import attention_ref, flash_attention, flash_attention_packed, flash_attention_varlen_packed
from .fused import (ce_loss_and_grad_, ce_stats, clamped_glu, cross_entropy, cross_entropy_ref, depth_residual, dyn_tanh_residual,
                    embedding, gelu_glu, gelu_lookup, grad_to_buf, merge_ce_stats, post_norm_step, rms_norm, rms_norm_ref, rope_qkv, rope_ref, rope_tables, silu_glu, swiglu,
                    swiglu_ref, swiglu_silu_gate)
from . import moe  # noqa: F401
from .delta import gated_delta
from .gemm import decode_linear, gemm_bf16, linear, matmul_nt, project, project_inputs, stream_linear
from .latent import latent_attention
from .paged import (decode_attention_gqa, paged_attention_ref, paged_decode_attention, paged_decode_attention_int8,
                    paged_decode_attention_mx,
                    paged_prefill_attention, paged_prefill_attention_int8, prefill_attention_gqa)
from .pre_norm import pre_norm_step
from .ragged import ragged_attention, shaped_attention
from .retention import retention
from .rglru import rglru
from .ssd import ssd
from .timemix import gated_linear, time_mix, token_shift

__all__ = [
    "attention_ref", "flash_attention", "flash_attention_packed", "flash_attention_varlen_packed", "ce_loss_and_grad_", "ce_stats", "cross_entropy", "cross_entropy_ref",
    "embedding", "grad_to_buf", "merge_ce_stats", "rms_norm", "rms_norm_ref", "rope_qkv", "rope_ref",
    "rope_tables", "swiglu", "swiglu_ref", "swiglu_silu_gate", "decode_linear", "stream_linear", "gemm_bf16", "linear", "matmul_nt", "decode_attention_gqa", "paged_attention_ref", "paged_decode_attention",
    "paged_decode_attention_int8", "paged_decode_attention_mx", "paged_prefill_attention", "paged_prefill_attention_int8", "prefill_attention_gqa",
    "clamped_glu", "depth_residual", "dyn_tanh_residual", "gated_delta", "latent_attention", "project", "ragged_attention", "retention", "rglru",
    "silu_glu", "gated_linear", "gelu_glu", "gelu_lookup", "post_norm_step", "pre_norm_step", "project_inputs", "shaped_attention", "ssd", "time_mix", "token_shift",
]
