// Parameters shared by the two forms of the generalised delta rule.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "../common/ragged.cuh"

namespace eredu {

template <typename T>
struct DeltaParams {
  const T* proj;           // [M, ld] = [r | k | v | output gate | removal rate | decay input]
  const float* w2;         // [H dk, rank]
  const float* w0;         // [H dk]
  const float* rate_b;     // [H dk]
  const float* norm_w;     // [H dv]
  float* state;            // [slots, H, dk, dv]
  T* out;                  // [M, H dv]
  int H, dk, dv, rank, ld;
  float log_decay, eps;
  RaggedBatch seqs;
};

constexpr float kUnitEps = 1e-6f;    // added to a key's squared length

// Chunk-parallel form for long bf16 portions (general_delta_chunk.cu): bytes of scratch it needs (0: not taken).
long long delta_chunk_bytes(int H, int dk, int dv, int rank, int rows, int batch, int max_rows);
bool delta_chunk_supported(const DeltaParams<__nv_bfloat16>& p);
cudaError_t launch_delta_chunks(const DeltaParams<__nv_bfloat16>& p, int max_rows, void* scratch, cudaStream_t stream);

}  // namespace eredu
