// Launcher of the persistent large-M tcgen05 GEMM (gemm_persistent.cu), called by eredu_gemm_bf16 for prefill-
// sized problems. Returns a cudaError_t, a negative tensor-map error, or kPersistentUnsupported when the problem
// does not meet the kernel's layout requirements (the caller then uses the one-tile-per-CTA kernel).
#pragma once
#include <cuda_runtime.h>

namespace eredu {

constexpr int kPersistentUnsupported = -7777;

int launch_gemm_persistent(const void* X, const void* W, void* Y, const void* residual, const void* bias, int M, int N,
                           int K, int ldx, int ldw, int ldy, int ldr, int w_rows, int dual, int dual_row_offset,
                           int sm_count, int* status, const float* ssq_in, int ssq_parts, float norm_eps, int norm_dim,
                           float* ssq_out, int act, float act_a, float act_b, int out_fp32, cudaStream_t stream);

// Expert GEMMs over a work table whose items have at most 256 rows (eredu_gemm_bf16_grouped with tile 256): no bias, SwiGLU when dual.
int launch_gemm_persistent_grouped(const void* X, const void* W, void* Y, const int* work, int n_work, int rows_cap, int N, int K, int ldx,
                                   int ldw, int ldy, int w_rows_total, int w_rows_per_expert, int dual, int sm_count, int* status,
                                   cudaStream_t stream);

}  // namespace eredu
