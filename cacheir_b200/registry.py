"""Backend registry entry for the B200 decode backend.

Same declarative shape as the reference registry (cacheir/backends/registry.py:6-67):
a `Backend` names its devices and the kernel-level names it provides. The op
names a compiled graph carries (`paged_attention_decode`, `quantized_matmul`,
`quantized_fused_rmsnorm_qkv_rope`, `quantized_fused_swiglu`, ...) and the
`attrs["kernel"]` strings written by the reference's `KernelSelection` pass
(cacheir/passes/transformer.py:356-388) are accepted unchanged; `KERNEL_FOR_OP`
records which C entry point serves each of them.
"""
from __future__ import annotations

from dataclasses import dataclass


@dataclass(frozen=True)
class Backend:
    name: str
    devices: tuple[str, ...]
    kernels: tuple[str, ...]
    notes: str = ""


class BackendRegistry:
    def __init__(self) -> None:
        self._backends: dict[str, Backend] = {}

    def register(self, backend: Backend) -> None:
        self._backends[backend.name] = backend

    def get(self, name: str) -> Backend:
        return self._backends[name]

    def names(self) -> list[str]:
        return sorted(self._backends)


# graph op  ->  (kernel name in attrs["kernel"] for cuda targets, C entry points that execute it)
KERNEL_FOR_OP: dict[str, tuple[str, tuple[str, ...]]] = {
    "token_embedding": ("triton.embedding_gather", ("cacheir_b200_embedding_gather",)),
    "rms_norm": ("triton.rms_norm", ("cacheir_b200_rms_norm",)),
    "matmul": ("triton.matmul_tensorcore", ("cacheir_b200_qgemv",)),
    "quantized_matmul": ("triton.awq_int4_tensorcore", ("cacheir_b200_qgemv",)),
    "fused_rmsnorm_qkv_rope": ("triton.fused_rmsnorm_qkv_rope",
                               ("cacheir_b200_rms_norm", "cacheir_b200_qgemv", "cacheir_b200_rope_inplace")),
    "quantized_fused_rmsnorm_qkv_rope": ("triton.awq_fused_rmsnorm_qkv_rope",
                                         ("cacheir_b200_rms_norm", "cacheir_b200_qgemv", "cacheir_b200_rope_inplace")),
    "paged_attention_decode": ("triton.paged_attention_decode",
                               ("cacheir_b200_kv_append", "cacheir_b200_paged_attention_decode_batch")),
    "fused_swiglu": ("triton.fused_swiglu", ("cacheir_b200_qgemv",)),
    "quantized_fused_swiglu": ("triton.awq_fused_swiglu", ("cacheir_b200_qgemv",)),
    "add": ("triton.vector_add", ("cacheir_b200_add", "cacheir_b200_qgemv")),
}

# graph ops of the ragged families -> C entry points of their libraries (tensor-core forms first)
HYBRID_KERNELS_FOR_OP: dict[str, tuple[str, ...]] = {
    "scaled_token_embedding": ("cacheir_b200_scaled_embedding",),
    "dynamic_tanh": ("cacheir_b200_dyt_rows",),
    "concat_matmul": ("cacheir_b200_dense_gemm", "cacheir_b200_dense_simple", "cacheir_b200_silu_cols"),
    "matmul": ("cacheir_b200_dense_gemm", "cacheir_b200_dense_simple", "cacheir_b200_relu2_cols"),
    "latent_attention": ("cacheir_b200_latent_prepare", "cacheir_b200_dense_gemm", "cacheir_b200_latent_attention",
                         "cacheir_b200_latent_attention_simple"),
    "linear_recurrence": ("cacheir_b200_recurrence_step", "cacheir_b200_recurrence_chunked", "cacheir_b200_recurrence_simple"),
    "gated_rms_norm": ("cacheir_b200_gated_rms",),
    "residual_dynamic_tanh": ("cacheir_b200_dense_gemm", "cacheir_b200_residual_dyt"),
    "fused_geglu": ("cacheir_b200_dense_gemm", "cacheir_b200_dense_simple", "cacheir_b200_glu_pairs"),
    "token_side_gate": ("cacheir_b200_dense_gemm", "cacheir_b200_dense_simple", "cacheir_b200_gelu_embed"),
    "residual_rms_norm": ("cacheir_b200_residual_rms",),
    "fused_glu": ("cacheir_b200_dense_gemm", "cacheir_b200_dense_simple", "cacheir_b200_glu_pairs"),
    "rms_norm": ("cacheir_b200_rms_rows",),
    "tied_attention": ("cacheir_b200_tied_prepare", "cacheir_b200_tied_attention_step", "cacheir_b200_tied_attention_prompt",
                       "cacheir_b200_tied_attention_simple"),
    "expert_router": ("cacheir_b200_dense_gemm", "cacheir_b200_dense_simple", "cacheir_b200_route"),
    "expert_mixture": ("cacheir_b200_grouped_gemm", "cacheir_b200_grouped_simple", "cacheir_b200_glu_pairs"),
    "combine_residual_rms_norm": ("cacheir_b200_combine_residual_rms",),
    "add_token_embedding": ("cacheir_b200_scaled_embedding",),
    "matrix_memory": ("cacheir_b200_memory_step", "cacheir_b200_memory_gates", "cacheir_b200_recurrence_chunked", "cacheir_b200_recurrence_simple",
                      "cacheir_b200_memory_norm"),
    "residual_add": ("cacheir_b200_residual_add",),
    "join_embedding": ("cacheir_b200_join_embedding", "cacheir_b200_dense_gemm", "cacheir_b200_dense_simple"),
    "layer_norm": ("cacheir_b200_layer_norm_rows",),
    "talking_attention": ("cacheir_b200_talking_prepare", "cacheir_b200_talking_step", "cacheir_b200_talking_prompt", "cacheir_b200_talking_simple"),
    "short_conv": ("cacheir_b200_short_conv",),
    "state_space": ("cacheir_b200_state_space_step", "cacheir_b200_state_space_gates", "cacheir_b200_recurrence_chunked", "cacheir_b200_recurrence_simple"),
    "delta_rule": ("cacheir_b200_delta_step", "cacheir_b200_delta_chunked", "cacheir_b200_delta_simple", "cacheir_b200_gated_parts_rms"),
    "gated_parts_rms": ("cacheir_b200_gated_parts_rms",),
    "residual_rms_pair": ("cacheir_b200_residual_rms_pair",),
    "combine_residual": ("cacheir_b200_combine_residual",),
}

B200_BACKEND = Backend(
    name="cuda-b200",
    devices=("sm100a",),
    kernels=(
        "embedding_gather",
        "rms_norm",
        "fused_rmsnorm_qkv_rope",
        "awq_fused_rmsnorm_qkv_rope",
        "paged_attention_decode",
        "paged_attention_decode_batch_splitk",
        "fused_swiglu",
        "awq_fused_swiglu",
        "awq_int4_tensorcore",
        "qgemv_int8",
        "qgemv_int4",
        "qgemv_int4_group128",
        "matmul_tensorcore",
        "kv_page_append",
        "quant_pack_rows",
        "cuda_graph_decode_replay",
        "dense_gemm_bf16",
        "latent_attention",
        "linear_recurrence",
        "tied_attention",
        "matrix_memory",
        "talking_attention",
        "state_space",
        "delta_rule",
        "short_conv",
        "grouped_gemm_bf16",
        "expert_routing",
    ),
    notes="Hand-written sm_100a kernels behind a C ABI (libcacheir_b200.so): split-K paged decode attention over a "
          "shared page pool, packed int4/int8 dequant-GEMV, fused glue ops; decode step replayed as a CUDA graph.",
)


def default_registry() -> BackendRegistry:
    registry = BackendRegistry()
    registry.register(B200_BACKEND)
    return registry
