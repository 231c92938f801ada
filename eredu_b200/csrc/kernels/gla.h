// Arguments of the gated linear attention kernels (gla.cu: token by token; gla_chunk.cu: long portions on the tensor cores).
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "../common/ragged.cuh"

namespace eredu {

template <typename T>
struct GlaParams {
  const T* proj;         // [M, ld] = [q (H dk) | k (H dk) | v (H dv) | gate (H dv) | low (rank)]
  const float* a2;       // [H dk, rank]
  const float* a2_b;     // [H dk]
  const float* norm_w;   // [dv]
  float* state;          // [slots, H, dk, dv]
  T* out;                // [M, H dv]
  int H, dk, dv, rank, ld;
  float inv_tau, eps;
  RaggedBatch seqs;
};

// Long portions (gla_chunk.cu). `ws` holds gla_chunk_count(rows, batch) matrices [H, dk, dv] and `decay` as many [H, dk].
bool gla_chunk_supported(const GlaParams<__nv_bfloat16>& p);
long long gla_chunk_count(int rows, int batch);
cudaError_t launch_gla_chunks(const GlaParams<__nv_bfloat16>& p, int max_rows, float* ws, float* decay, cudaStream_t stream);

}  // namespace eredu
