// Gated linear attention: a matrix state per head with a decay per key channel.
//   alpha_t = sigmoid(z_t)^(1 / tau), z_t = A2 low_t + bias      (low_t: the rank-r part of the projection)
//   S_t = diag(alpha_t) S_{t-1} + k_t v_t^T,  o_t = S_t^T q_t / sqrt(dk),  y_t = w rms-norm(o_t) silu(gate_t)
// proj [M, 2 H dk + 2 H dv + r] = [q | k | v | gate | low]; S fp32 [slots, H, dk, dv]. Decays, scores and S are fp32.
#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/launch_count.h"
#include "../common/ptx.cuh"
#include "../common/ragged.cuh"
#include "gla.h"

namespace eredu {

// Decode steps and short portions, any size, bf16 or fp32: one CTA per (head, sequence). The state streams through
// registers once per token (VEC columns per load); row groups of the block share the dk rows and meet in shared memory for
// o, which is normalised, gated and stored by the same CTA. The decays of the head are formed from the low-rank input here,
// so a decode step of the layer is this launch between its two projections.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) gla_step_kernel(GlaParams<T> p) {
  extern __shared__ float sm[];
  __shared__ float red[8];
  pdl_launch_early();
  const int dk = p.dk, dv = p.dv;
  float* qs = sm;               // [dk] query / sqrt(dk)
  float* ks = qs + dk;          // [dk]
  float* as = ks + dk;          // [dk] decay
  float* lows = as + dk;        // [rank]
  float* os = lows + p.rank;    // [row groups][dv]
  const int h = blockIdx.x;
  if (p.seqs.cu_q == nullptr && (dv & 3) == 0) {
    // Decode: the state is not touched by the projection in front of this launch, so it starts towards L2 before the wait
    // (a row that turns out idle wastes a fetch of slot 0).
    const int slot = p.seqs.page_to_slot[p.seqs.block_table[static_cast<size_t>(blockIdx.y) * p.seqs.max_pages]];
    const char* base = reinterpret_cast<const char*>(p.state + (static_cast<size_t>(slot) * p.H + h) * dk * dv);
    const size_t bytes = static_cast<size_t>(dk) * dv * sizeof(float);
    for (size_t o = threadIdx.x * 1024; o < bytes; o += 256 * 1024)
      bulk_prefetch_l2(base + o, static_cast<uint32_t>(bytes - o < 1024 ? bytes - o : 1024));
  }
  pdl_wait();
  pdl_launch_dependents();
  const RaggedSeq s = ragged_seq(p.seqs, blockIdx.y);
  if (s.rows <= 0) return;  // uniform
  const int qk = p.H * dk, vw = p.H * dv;
  float* st = p.state + (static_cast<size_t>(s.slot) * p.H + h) * dk * dv;
  const int cols = dv / VEC;
  const int per_row = min(cols, 256);
  const int groups = 256 / per_row;
  const int grp = threadIdx.x / per_row, c_first = threadIdx.x % per_row;
  const float q_scale = 1.f / sqrtf(static_cast<float>(dk));
  for (int t = 0; t < s.rows; ++t) {
    const size_t m = static_cast<size_t>(s.row0 + t);
    const T* row = p.proj + m * p.ld;
    for (int i = threadIdx.x; i < p.rank; i += 256) lows[i] = to_f32(row[2 * qk + 2 * vw + i]);
    __syncthreads();
    for (int i = threadIdx.x; i < dk; i += 256) {
      qs[i] = to_f32(row[h * dk + i]) * q_scale;
      ks[i] = to_f32(row[qk + h * dk + i]);
      const float* a2 = p.a2 + static_cast<size_t>(h * dk + i) * p.rank;
      float z = p.a2_b[h * dk + i];
      if ((p.rank & 3) == 0) {
#pragma unroll 4
        for (int j = 0; j < p.rank; j += 4) {
          const float4 w = load4(a2 + j);
          z = fmaf(w.x, lows[j], fmaf(w.y, lows[j + 1], fmaf(w.z, lows[j + 2], fmaf(w.w, lows[j + 3], z))));
        }
      } else {
        for (int j = 0; j < p.rank; ++j) z = fmaf(a2[j], lows[j], z);
      }
      as[i] = expf(log_sigmoid_f32(z) * p.inv_tau);
    }
    __syncthreads();
    if (grp < groups) {
      for (int c = c_first; c < cols; c += per_row) {
        float v[VEC], o[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          v[e] = to_f32(row[2 * qk + h * dv + c * VEC + e]);
          o[e] = 0.f;
        }
#pragma unroll 8
        for (int r = grp; r < dk; r += groups) {
          float* cell = st + static_cast<size_t>(r) * dv + c * VEC;
          float x[VEC];
          if constexpr (VEC == 4) {
            const float4 f = s.live ? load4(cell) : make_float4(0.f, 0.f, 0.f, 0.f);
            x[0] = f.x, x[1] = f.y, x[2] = f.z, x[3] = f.w;
          } else {
            x[0] = s.live ? *cell : 0.f;
          }
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            x[e] = as[r] * x[e] + ks[r] * v[e];
            o[e] = fmaf(x[e], qs[r], o[e]);
          }
          if (s.live) {
            if constexpr (VEC == 4) store4(cell, make_float4(x[0], x[1], x[2], x[3]));
            else *cell = x[0];
          }
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) os[grp * dv + c * VEC + e] = o[e];
      }
    }
    __syncthreads();
    float ss = 0.f;
    for (int j = threadIdx.x; j < dv; j += 256) {
      float o = 0.f;
      for (int g = 0; g < groups; ++g) o += os[g * dv + j];
      os[j] = o;
      ss += o * o;
    }
    const float inv = 1.f / sqrtf(block_sum_f32(ss, red) / static_cast<float>(dv) + p.eps);
    for (int j = threadIdx.x; j < dv; j += 256) {
      const float g = to_f32(row[2 * qk + vw + h * dv + j]);
      p.out[m * vw + h * dv + j] = from_f32<T>(os[j] * inv * p.norm_w[j] * silu_f32(g));
    }
    __syncthreads();
  }
}

constexpr int kGlaChunkMinRows = 16;  // from this portion length on the chunk-parallel form takes over

template <typename T>
static cudaError_t launch_gla_step(const GlaParams<T>& p, cudaStream_t stream) {
  const int vec = p.dv % 4 == 0 ? 4 : 1;
  const int cols = p.dv / vec, per_row = cols < 256 ? cols : 256;
  const size_t smem = (static_cast<size_t>(3) * p.dk + p.rank + static_cast<size_t>(256 / per_row) * p.dv) * sizeof(float);
  if (smem > 48 * 1024) return cudaErrorInvalidValue;
  const dim3 grid(p.H, p.seqs.B);
  return vec == 4 ? launch_pdl(gla_step_kernel<T, 4>, grid, dim3(256), smem, stream, p)
                  : launch_pdl(gla_step_kernel<T, 1>, grid, dim3(256), smem, stream, p);
}

}  // namespace eredu

using namespace eredu;

// fp32 elements of scratch a bf16 call over `rows` rows of `batch` sequences can use (0: the token-by-token kernel serves it).
extern "C" long long eredu_gla_scratch_elems(int heads, int dk, int dv, int rank, int ld, int rows, int batch, int max_rows) {
  GlaParams<__nv_bfloat16> p = {};
  p.H = heads;
  p.dk = dk;
  p.dv = dv;
  p.rank = rank;
  p.ld = ld;
  if (max_rows < kGlaChunkMinRows || !gla_chunk_supported(p)) return 0;
  return gla_chunk_count(rows, batch) * heads * dk * (static_cast<long long>(dv) + 1);
}

// scratch: fp32 [eredu_gla_scratch_elems(...)] of a bf16 call over `rows` rows, or null (token by token).
extern "C" int eredu_gla_scan(const void* proj, const float* a2, const float* a2_b, const float* norm_w, float* state, void* out,
                              float* scratch, int rows, const int* block_table, const int* page_to_slot, const int* cu_q, const long long* slots, int heads,
                              int dk, int dv, int rank, int ld, int batch, int q_per_seq, int max_rows, int max_pages, int fp32,
                              float tau, float eps, cudaStream_t stream) {
  if (batch <= 0 || max_rows <= 0) return 0;
  if (heads <= 0 || dk <= 0 || dv <= 0 || rank <= 0 || tau <= 0.f) return -1;
  const RaggedBatch r = {block_table, page_to_slot, cu_q, slots, batch, q_per_seq, max_pages};
  cudaError_t e;
  if (fp32) {
    GlaParams<float> p = {static_cast<const float*>(proj), a2, a2_b, norm_w, state, static_cast<float*>(out), heads, dk, dv, rank, ld,
                          1.f / tau, eps, r};
    e = launch_gla_step(p, stream);
  } else {
    GlaParams<__nv_bfloat16> p = {static_cast<const __nv_bfloat16*>(proj), a2, a2_b, norm_w, state, static_cast<__nv_bfloat16*>(out),
                                  heads, dk, dv, rank, ld, 1.f / tau, eps, r};
    if (scratch != nullptr && max_rows >= kGlaChunkMinRows && gla_chunk_supported(p)) {
      float* decay = scratch + gla_chunk_count(rows, batch) * heads * dk * dv;
      e = launch_gla_chunks(p, max_rows, scratch, decay, stream);
      eredu_count_launches(2);
    } else {
      e = launch_gla_step(p, stream);
    }
  }
  eredu_count_launches(1);
  return static_cast<int>(e);
}
