"""Python wrappers over the sm_100a kernel library (tensors in, tensors out, current CUDA stream)."""
from .attention import (Differential, chunk_attention, dense_attention, dense_attention_padded, exchange_attention, exchange_decode_fits,  # noqa: F401
                        narrow_heads_on_kernel, paged_attention, varlen_causal_attention)
from .gemm import SSQ_WORDS, ssq_buffer, ssq_values, gemm_bf16, gemm_bf16_grouped, gemm_bf16_normed, gemm_f32, gated_fused, gemm_workspace, linear, linear_gated  # noqa: F401
from .llm import (argmax, sample_device, embedding, gated_act_mul, gated_residual, layernorm_mod, poly_norm, rmsnorm, rope_kv_write, row_rope_kv_write, diff_combine, head_mix, head_mix_weights,  # noqa: F401
                  spec_verify_greedy)
from .delta import DeltaWeights, channel_delta, delta_key_width, head_delta  # noqa: F401
from .hyper import HyperBranch, ShortConv, StreamMix, hyper_step, short_conv  # noqa: F401
from .latent import (LatentWeights, QueryRotation, SplitPartials, head_product, latent_attention_simple, latent_decode, latent_decode_supported,  # noqa: F401
                     latent_gather, latent_prefill, latent_prefill_supported, latent_prep, latent_width, rotate_queries)
from .moe import RoutingPlan, gemm_grouped_rows, logits_routing, routed_ffn, routed_gated_ffn, table_routing  # noqa: F401
from .stream import Branch, DepthAverage, NormWeights, RoutedRows, stream_embed, stream_embed_pairs, stream_norm  # noqa: F401
from .runtime import KernelError, check_status, device_status  # noqa: F401
from .dit import axpy, conv3x3_nhwc, conv3x3_supported, groupnorm_nhwc, im2col3x3_nhwc, rgb8_nhwc, softmax_rows, upsample2x_nhwc  # noqa: E402,F401
from .quant import QuantWeight, dequantize, linear_any, linear_quant, quantize_weight  # noqa: E402,F401
