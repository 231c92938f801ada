"""Operators of the runtime: sm_100a kernels for CUDA tensors, PyTorch references for CPU tensors."""
from .core import (CLUSTER_SPLITS, KERNEL_HEAD_DIMS, PAGE, XIELU, attention_decode, attention_decode_rope, attention_prefill, attention_ref, branch_norm, branch_norm_ref, decode_scratch, decode_splits, embedding,
                   embedding_stream, gated_linear, gated_linear_ref, linear, linear_ref, qkv_prepare, qkv_prepare_ref, residual_norm,
                   residual_norm_ref, rms_residual, rms_residual_ref, rmsnorm, rmsnorm_ref, rope_kv, rope_kv_ref, silu_mul)
from .sampling import (SamplingParams, pack_allow_mask, pack_rows, philox_uniform, process_logits_ref, rows_to_tensor,
                       sample, sample_ref, spec_verify, verify_ref)
from .conv import (ConvChannels, ConvHeads, StreamConv, conv_project, conv_project_ref, short_conv, short_conv_ref, stream_conv,
                   stream_conv_ref)
from .recurrent import (gated_delta_scan, gated_delta_scan_ref, gla_attention, gla_attention_ref, gla_scan_ref, general_delta, general_delta_ref, general_delta_scan_ref, mamba2_scan,
                        mamba2_scan_ref, mingru_scan, mingru_scan_ref, mlstm, mlstm_ref, mlstm_scan_ref, mlstm_state_views,
                        selective_scan, selective_scan_ref)
from .pooling import blocks_seen, gather_pooled, pool_block_ref, pool_blocks, pool_cached_blocks, pooled_attention, pooled_attention_ref, pooled_row
from .latent import head_linear, latent_attention, latent_attention_ref, latent_prepare, latent_prepare_ref
from .talking import talking_attention, talking_attention_ref
from . import native
