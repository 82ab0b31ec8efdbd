"""B200-native (sm_100a) self-speculative verify step for looped language models.

Hand-written CUDA kernels behind a C ABI (``include/rlt_verify.h``,
``vllm_rlt_b200/librlt_verify.so``) plus the thin PyTorch host layer that mirrors the
attention-backend, sampler, speculative and ``torch.ops.vllm_rlt`` interfaces of vllm-rlt
for this one path.  There is no CPU or library fallback: importing is cheap, the first call
raises if the CUDA library has not been built.
"""

from ._capi import NativeLibraryMissing, load as load_library
from .activation import register_torch_op, silu_and_mul, silu_and_mul_packed
from .attention import (B200_CAPABILITIES, AttentionBackend, B200PagedAttention, BackendCapabilities,
                        ScoreTerms, create_backend)
from .checkpoint import read_safetensors, read_weights
from .decoder import DecodeStats, GraphedLoops, PagedKV, SelfSpeculativeDecoder
from .prefix_cache import PrefixIndex
from .engine import Engine, StepEntry
from .hybrid_lm import HybridLM, HybridLMConfig
from .kv_cache import RollbackResult, finalize_tokens, kv_write, rollback
from .experts import expert_gather, expert_gemm, expert_route, paired_rows
from .latent import (YarnScaling, latent_gather, latent_prompt_attention, latent_prompt_supported, latent_write, packed_attention,
                     rotate_heads, rotation_frequencies)
from .layers import (block_epilogue, clamped_glu, gated_unit, head_gate, head_mix, norm_rotate, residual_norm, rope_kv_write, sandwich_norm,
                     soft_cap, stream_mix)
from .looped_lm import LoopedLM, LoopedLMConfig, seeded_state_dict
from .postnorm_lm import PostNormLM, PostNormLMConfig
from .recurrent import causal_conv, conv_heads, decay_scan, decay_table, delta_scan, gated_norm, ssd_scan
from .registry import load_model, register_model, registered_architectures
from .runner import (B200SpeculativeRunner, KVCacheManagerView, ModelRunnerOutput, Request, SamplingParams, ScheduledRequest,
                     SchedulerOutput, SpeculativeConfig, SpeculativeRoundTicket, SpeculativeStats)
from .sandwich_lm import SandwichLM, SandwichLMConfig
from .stream_lm import StreamLM, StreamLMConfig
from .talking_mixer import talking_attention, talking_decode, talking_prompt
from .sequence_cache import CacheFull, CacheSpec, KVSpec, SequenceCache, StateSpec
from .speculative import (PipelineState, SpeculativeResult, accept_greedy, accept_rejection, argmax_rows,
                          decode_result, pipeline_shift, probabilities, raise_for_status, round_uniforms,
                          sample_rows)

__all__ = [
    "AttentionBackend", "B200PagedAttention", "DecodeStats", "GraphedLoops", "LoopedLM", "LoopedLMConfig", "PagedKV", "PrefixIndex",
    "SelfSpeculativeDecoder", "seeded_state_dict", "B200_CAPABILITIES", "BackendCapabilities",
    "NativeLibraryMissing", "RollbackResult", "SpeculativeResult", "accept_greedy", "accept_rejection",
    "argmax_rows", "PipelineState", "create_backend", "decode_result", "finalize_tokens", "pipeline_shift", "kv_write", "load_library", "probabilities", "raise_for_status",
    "register_torch_op", "rollback", "rope_kv_write", "sample_rows", "sandwich_norm", "silu_and_mul",
    "B200SpeculativeRunner", "ModelRunnerOutput", "Request", "SamplingParams", "ScheduledRequest", "SchedulerOutput",
    "SpeculativeConfig", "SpeculativeRoundTicket", "SpeculativeStats", "round_uniforms", "silu_and_mul_packed",
    "KVCacheManagerView", "CacheFull", "CacheSpec", "Engine", "HybridLM", "HybridLMConfig", "KVSpec", "ScoreTerms",
    "SequenceCache", "StateSpec", "StepEntry", "block_epilogue", "causal_conv", "gated_norm", "load_model", "read_safetensors",
    "read_weights", "register_model", "registered_architectures", "residual_norm", "ssd_scan",
    "StreamLM", "StreamLMConfig", "clamped_glu", "decay_scan", "decay_table", "expert_gather", "expert_gemm", "expert_route",
    "latent_gather", "latent_prompt_attention", "latent_prompt_supported", "latent_write", "rotate_heads", "rotation_frequencies", "stream_mix",
    "SandwichLM", "SandwichLMConfig", "YarnScaling", "conv_heads", "gated_unit", "head_gate", "packed_attention", "soft_cap",
    "PostNormLM", "PostNormLMConfig", "delta_scan", "head_mix", "norm_rotate", "paired_rows",
    "talking_attention", "talking_decode", "talking_prompt",
]
