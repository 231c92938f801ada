// minGRU recurrence: gates that read only the current token, a linear recurrence per channel, an output gate.
//   z = sigmoid(proj_z), c = u + 1/2 (u >= 0) or sigmoid(u) (u < 0), S <- (1 - z) S + z c, y = S silu(g)
// proj [M, 3 width] = [z | u | g]; S fp32 [slots, width]. All gate arithmetic and S are fp32.
//
// Because a step is affine in S, a segment of tokens is one affine map: long portions are cut into segments that are
// composed in parallel (a thread holds one channel of one segment in registers), the maps are chained through shared
// memory, and every segment is then replayed from its entering state. One pass over the inputs.
#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/launch_count.h"
#include "../common/ptx.cuh"
#include "../common/ragged.cuh"

namespace eredu {

template <typename T>
struct MinGruParams {
  const T* proj;
  float* state;
  T* out;
  int width, ld;
  RaggedBatch seqs;
};

// a step of the recurrence as S -> a S + b
__device__ __forceinline__ void mingru_step(float z_in, float u, float& a, float& b) {
  const float z = sigmoid_f32(z_in);
  a = 1.f - z;
  b = z * (u >= 0.f ? u + 0.5f : sigmoid_f32(u));
}

// Decode steps and short portions: one thread per channel, token after token.
template <typename T>
__global__ void __launch_bounds__(128) mingru_step_kernel(MinGruParams<T> p) {
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const RaggedSeq s = ragged_seq(p.seqs, blockIdx.y);
  const int c = blockIdx.x * 128 + threadIdx.x;
  if (c >= p.width || s.rows <= 0) return;
  float* st = p.state + static_cast<size_t>(s.slot) * p.width + c;
  float S = s.live ? *st : 0.f;
  for (int t = 0; t < s.rows; ++t) {
    const T* r = p.proj + static_cast<size_t>(s.row0 + t) * p.ld + c;
    float a, b;
    mingru_step(to_f32(r[0]), to_f32(r[p.width]), a, b);
    S = a * S + b;
    p.out[static_cast<size_t>(s.row0 + t) * p.width + c] = from_f32<T>(S * silu_f32(to_f32(r[2 * p.width])));
  }
  if (s.live) *st = S;
}

constexpr int kSegs = 16;   // segments a tile is cut into
constexpr int kSegLen = 8;  // tokens of a segment
constexpr int kTileTokens = kSegs * kSegLen;

template <typename T>
__global__ void __launch_bounds__(32 * kSegs) mingru_scan_kernel(MinGruParams<T> p) {
  __shared__ float sa[kSegs][32], sb[kSegs][32], carry[32];
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const RaggedSeq s = ragged_seq(p.seqs, blockIdx.y);
  if (s.rows <= 0) return;  // uniform
  const int lane = threadIdx.x & 31, seg = threadIdx.x >> 5;
  const int c = blockIdx.x * 32 + lane;
  const bool in = c < p.width;
  float* st = p.state + static_cast<size_t>(s.slot) * p.width + (in ? c : 0);
  if (seg == 0) carry[lane] = in && s.live ? *st : 0.f;
  T zr[kSegLen], ur[kSegLen], gr[kSegLen];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < kSegLen; ++i) {
      const int t = t0 + seg * kSegLen + i;
      if (in && t < s.rows) {
        const T* r = p.proj + static_cast<size_t>(s.row0 + t) * p.ld + c;
        zr[i] = r[0];
        ur[i] = r[p.width];
        gr[i] = r[2 * p.width];
      } else {
        zr[i] = ur[i] = gr[i] = from_f32<T>(0.f);
      }
    }
  };
  fetch(0);
  for (int t0 = 0; t0 < s.rows; t0 += kTileTokens) {
    float a[kSegLen], b[kSegLen], g[kSegLen];
    float A = 1.f, B = 0.f;
#pragma unroll
    for (int i = 0; i < kSegLen; ++i) {
      if (t0 + seg * kSegLen + i < s.rows) mingru_step(to_f32(zr[i]), to_f32(ur[i]), a[i], b[i]);
      else a[i] = 1.f, b[i] = 0.f;  // behind the portion: the state stays
      g[i] = silu_f32(to_f32(gr[i]));
      A *= a[i];
      B = a[i] * B + b[i];
    }
    if (t0 + kTileTokens < s.rows) fetch(t0 + kTileTokens);  // in flight while the segments are chained
    sa[seg][lane] = A;
    sb[seg][lane] = B;
    __syncthreads();
    float S = carry[lane];
    for (int j = 0; j < seg; ++j) S = sa[j][lane] * S + sb[j][lane];
    __syncthreads();  // every thread has read the carry and the maps of this tile
#pragma unroll
    for (int i = 0; i < kSegLen; ++i) {
      const int t = t0 + seg * kSegLen + i;
      S = a[i] * S + b[i];
      if (in && t < s.rows) p.out[static_cast<size_t>(s.row0 + t) * p.width + c] = from_f32<T>(S * g[i]);
    }
    if (seg == kSegs - 1) carry[lane] = S;
  }
  __syncthreads();
  if (seg == 0 && in && s.live) *st = carry[lane];
}

template <typename T>
static cudaError_t launch_mingru(const MinGruParams<T>& p, int max_rows, cudaStream_t stream) {
  if (max_rows <= 8) return launch_pdl(mingru_step_kernel<T>, dim3((p.width + 127) / 128, p.seqs.B), dim3(128), 0, stream, p);
  return launch_pdl(mingru_scan_kernel<T>, dim3((p.width + 31) / 32, p.seqs.B), dim3(32 * kSegs), 0, stream, p);
}

}  // namespace eredu

using namespace eredu;

extern "C" int eredu_mingru_scan(const void* proj, float* state, void* out, const int* block_table, const int* page_to_slot,
                                 const int* cu_q, const long long* slots, int width, int ld, int batch, int q_per_seq, int max_rows,
                                 int max_pages, int fp32, cudaStream_t stream) {
  if (batch <= 0 || width <= 0 || max_rows <= 0) return 0;
  const RaggedBatch r = {block_table, page_to_slot, cu_q, slots, batch, q_per_seq, max_pages};
  cudaError_t e;
  if (fp32) {
    MinGruParams<float> p = {static_cast<const float*>(proj), state, static_cast<float*>(out), width, ld, r};
    e = launch_mingru(p, max_rows, stream);
  } else {
    MinGruParams<__nv_bfloat16> p = {static_cast<const __nv_bfloat16*>(proj), state, static_cast<__nv_bfloat16*>(out), width, ld, r};
    e = launch_mingru(p, max_rows, stream);
  }
  eredu_count_launches(1);
  return static_cast<int>(e);
}
