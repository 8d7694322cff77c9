"""Operators.  Every op has two implementations selected by the input's device:

* CUDA tensors run the hand-written sm_100a kernels from ``csrc/`` (there is no PyTorch fallback on a
  GPU: a missing kernel library raises);
* CPU tensors run a plain PyTorch fp32-accurate implementation, which is the numerical oracle of the
  test-suite and the path used by the gloo plumbing tests.
"""
from .gemm import gemm, linear, linear_act, lora_linear, grad_into_main
from .elementwise import rmsnorm, qknorm_rope, qknorm_rope_store, swiglu, embedding, rope_tables
from .attention import flash_attention
from .loss import lm_head_cross_entropy, lm_head_logprob, grpo_token_loss, VocabShard, valid_rows
from .optim import sumsq, fused_adamw
from .paged import (kv_store, kv_gather, paged_decode_attention, paged_prefill_attention, varlen_attention,
                    topp_sample)
from .residual import (embedding_f32, embedding_pairs, rmsnorm_f32, layernorm_f32, merge_norm_add, norm_add, branch_add, post_norm, glu,
                       gelu_times_token, rope_rows, rope_turns)
from .linear_state import retention, delta_inputs, gated_delta, matrix_memory
from .recurrence import gated_recurrence, causal_conv, block_gates, linear_recurrence
from .moe import Routing, route, router, linear_fp32, token_gate, glu_linear, expert_glu, expert_down, moe_norm_add
from .paged_rows import qk_norm_store, paged_attention, differential_attention, distance_buckets
from .latent import latent_store, latent_turn, latent_attention, latent_rows, head_linear

__all__ = [
    "gemm", "linear", "linear_act", "lora_linear", "grad_into_main", "rmsnorm", "qknorm_rope", "qknorm_rope_store", "swiglu", "embedding", "rope_tables",
    "flash_attention", "VocabShard", "valid_rows", "lm_head_cross_entropy", "lm_head_logprob", "grpo_token_loss", "sumsq",
    "fused_adamw", "kv_store", "kv_gather", "paged_decode_attention", "paged_prefill_attention", "varlen_attention", "topp_sample",
    "embedding_f32", "embedding_pairs", "rmsnorm_f32", "layernorm_f32", "merge_norm_add", "branch_add", "post_norm", "glu", "rope_rows", "rope_turns", "retention", "delta_inputs",
    "gated_delta", "matrix_memory", "gated_recurrence", "causal_conv", "block_gates", "linear_recurrence", "Routing", "route", "router", "linear_fp32", "token_gate", "glu_linear", "expert_glu", "expert_down",
    "moe_norm_add", "norm_add", "gelu_times_token", "qk_norm_store", "paged_attention", "differential_attention", "distance_buckets",
    "latent_store", "latent_turn", "latent_attention", "latent_rows", "head_linear",
]
