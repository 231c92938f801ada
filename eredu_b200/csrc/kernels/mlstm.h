// Arguments of the mLSTM kernels (mlstm.cu: token by token; mlstm_chunk.cu: long portions on the tensor cores).
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "../common/elem.cuh"
#include "../common/ragged.cuh"

namespace eredu {

template <typename T>
struct MlstmParams {
  const T* proj;         // [M, ld] = [q (H dk) | k (H dk) | v (H dv) | output gate (H dv)]
  const float* gates;    // [M, ldg] = [input (H) | forget (H)] pre-activations
  const float* norm_w;   // [H dv]
  float* state;          // [slots, stride]: memory [H, dk, dv], normaliser [H, dk], running maximum [H]
  T* out;                // [M, H dv]
  int H, dk, dv, ld, ldg;
  long long stride;
  float cap, eps;
  RaggedBatch seqs;
};

constexpr float kMlstmEps = 1e-6f;   // added to the normaliser

// Log input gate and log forget gate of one token and head.
__device__ __forceinline__ float2 mlstm_gates(const float* gates, int H, int h, float cap) {
  const float zi = cap * tanhf(gates[h] / cap), zf = cap * tanhf(gates[H + h] / cap);
  return make_float2(zi, log_sigmoid_f32(zf));
}

// Long portions. `ws`: scratch of mlstm_chunk_bytes(...).
bool mlstm_chunk_supported(int dk, int dv, int ld, long long stride);
long long mlstm_chunk_bytes(int H, int dk, int dv, int rows, int batch);
cudaError_t launch_mlstm_chunks(const MlstmParams<__nv_bfloat16>& p, int rows, int max_rows, void* ws, cudaStream_t stream);

}  // namespace eredu
