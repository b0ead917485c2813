"""Hot-path operators: each one is a thin launcher around a hand-written sm_100a kernel
(with an f32 PyTorch evaluation of the same math for CPU tensors, used as the test oracle)."""
from .gemm import gemm, linear, linear_master, matmul_exact, mv, dot, bmm
from .norm import rms_norm, layer_norm, rmsnorm_fwd, rmsnorm_bwd
from .llama import (rope_tables, rope_inplace, apply_rope, swiglu, swiglu_fwd, swiglu_bwd, embedding, embedding_fwd,
                    embedding_bwd, add_)
from .loss import cross_entropy, cross_entropy_fwd_bwd
from .optim import adamw_flat_, sgd_flat_, grad_norm_, scale_
from .attention import attention_packed, flash_fwd, flash_bwd
from .streams import DynamicTanhWeights, HyperWeights, SublayerOutput, dynamic_tanh, hyper_embed, hyper_update
from .moe import ExpertStack, MoeWeights, MoeSmallBuffers, MoeRouting, RouteRule, moe_rows, moe_small, gated_act, grouped_linear, interleave_gate_up
from .latent_attention import (LatentDims, LatentWeights, LatentDecodeBuffers, latent_context, latent_attention_rows, latent_attention_decode, absorb_queries, expand_values,
                               rotary_pair_tables)
from .residual import (DenseGatedWeights, DensePolyWeights, TokenShift, dense_poly_rows, depth_embed, depth_update, poly_norm_planes, poly_norm_rows, token_shift, dense_gated_rows, gated_act_planes, gated_act_rows, parallel_embed, parallel_update, residual_embed,
                       residual_update)
from .gqa_attention import GqaDims, GqaWeights, GqaDecodeBuffers, gqa_attention_rows, gqa_attention_decode, pack_head_rows, pack_head_columns, pack_head_vector, differential_blend
from .matrix_memory import MemoryDims, MemoryWeights, matrix_memory_rows, matrix_memory_decode
from .state_space import SsmDims, SsmWeights, SsmDecodeBuffers, state_space_rows, state_space_decode
from . import attention

__all__ = [n for n in dir() if not n.startswith("_")]
from . import tensor_ops  # noqa: E402
from . import nn_ops  # noqa: E402
from . import conv  # noqa: E402
from .conv import conv3x3, conv3x3_nhwc_raw  # noqa: E402
