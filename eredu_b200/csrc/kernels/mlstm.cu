// mLSTM: a matrix memory per head with exponential gates, kept in range by a running maximum m of the log scale.
//   i_t = cap tanh(zi / cap), f_t = log sigmoid(cap tanh(zf / cap)), m_t = max(f_t + m_{t-1}, i_t)
//   S_t = e^(f_t + m_{t-1} - m_t) S_{t-1} + e^(i_t - m_t) k_t v_t^T,  n_t likewise with k_t alone
//   o_t = S_t^T q_t / (max(|n_t . q_t|, e^-m_t) + 1e-6),  y_t = w rms-norm(o_t) sigmoid(gate_t),  q scaled by dk^-1/2
// State fp32: S [H, dk, dv] | n [H, dk] | m [H]; all start at zero.
#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/launch_count.h"
#include "../common/ptx.cuh"
#include "../common/ragged.cuh"
#include "mlstm.h"

namespace eredu {

__device__ __forceinline__ float ld_cluster_f32(uint32_t addr) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
  return v;
}

// Decode steps and short portions, any size, bf16 or fp32. grid (column slices, heads, sequences); the slices of a head form a cluster
// and share the sum of squares of its output. A CTA keeps n and m, streams its columns of S through registers once per token (VEC
// columns per load; row groups of the block meet in shared memory), normalises, gates and stores.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) mlstm_step_kernel(MlstmParams<T> p) {
  extern __shared__ float sm[];
  __shared__ float red[8];
  __shared__ float s_ss[2];                      // this slice's sum of squares, by parity of the token
  pdl_launch_early();
  const int dk = p.dk, dv = p.dv, slices = gridDim.x;
  const int width = dv / slices, col0 = blockIdx.x * width;
  float* qs = sm;               // [dk] query / sqrt(dk)
  float* ks = qs + dk;          // [dk] key times its gate
  float* ns = ks + dk;          // [dk] normaliser
  float* os = ns + dk;          // [row groups][width]
  const int h = blockIdx.y;
  const size_t head_off = static_cast<size_t>(h) * dk * dv;
  if (p.seqs.cu_q == nullptr && VEC == 4) {
    // Decode: the state is not touched by the projection in front of this launch, so it starts towards L2 before the wait
    // (a row that turns out idle wastes a fetch of slot 0).
    const int slot = p.seqs.page_to_slot[p.seqs.block_table[static_cast<size_t>(blockIdx.z) * p.seqs.max_pages]];
    const float* base = p.state + slot * p.stride + head_off + col0;
    for (int r = threadIdx.x; r < dk; r += 256) bulk_prefetch_l2(base + static_cast<size_t>(r) * dv, width * 4);
  }
  pdl_wait();
  pdl_launch_dependents();
  const RaggedSeq s = ragged_seq(p.seqs, blockIdx.z);
  if (s.rows <= 0) return;      // uniform over the cluster
  const int qk = p.H * dk, vw = p.H * dv;
  if (!s.live) {                // an idle row: its result is not looked at, its state stays
    for (int t = 0; t < s.rows; ++t)
      for (int j = threadIdx.x; j < width; j += 256)
        p.out[static_cast<size_t>(s.row0 + t) * vw + h * dv + col0 + j] = from_f32<T>(0.f);
    return;
  }
  float* base = p.state + s.slot * p.stride;
  float* st = base + head_off + col0;
  float* n_state = base + static_cast<size_t>(p.H) * dk * dv + static_cast<size_t>(h) * dk;
  float* m_state = base + static_cast<size_t>(p.H) * dk * (dv + 1) + h;
  for (int i = threadIdx.x; i < dk; i += 256) ns[i] = n_state[i];
  float m = *m_state;
  const int cols = width / VEC;
  const int per_row = min(cols, 256);
  const int groups = 256 / per_row;
  const int grp = threadIdx.x / per_row, c_first = threadIdx.x % per_row;
  const float q_scale = 1.f / sqrtf(static_cast<float>(dk));
  for (int t = 0; t < s.rows; ++t) {
    const size_t row_i = static_cast<size_t>(s.row0 + t);
    const T* row = p.proj + row_i * p.ld;
    const float2 gt = mlstm_gates(p.gates + row_i * p.ldg, p.H, h, p.cap);
    const float m_new = fmaxf(gt.y + m, gt.x);
    const float keep = expf(gt.y + m - m_new), take = expf(gt.x - m_new);
    m = m_new;
    float dot = 0.f;
    for (int i = threadIdx.x; i < dk; i += 256) {
      const float q = to_f32(row[h * dk + i]) * q_scale, k = to_f32(row[qk + h * dk + i]) * take;
      const float n = fmaf(keep, ns[i], k);
      qs[i] = q;
      ks[i] = k;
      ns[i] = n;
      dot = fmaf(n, q, dot);
    }
    const float nq = block_sum_f32(dot, red);    // the barriers inside also publish qs and ks
    const float inv_den = 1.f / (fmaxf(fabsf(nq), expf(-m)) + kMlstmEps);
    if (grp < groups) {
      for (int c = c_first; c < cols; c += per_row) {
        float v[VEC], o[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          v[e] = to_f32(row[2 * qk + h * dv + col0 + c * VEC + e]);
          o[e] = 0.f;
        }
#pragma unroll 8
        for (int r = grp; r < dk; r += groups) {
          float* cell = st + static_cast<size_t>(r) * dv + c * VEC;
          float x[VEC];
          if constexpr (VEC == 4) {
            const float4 f = load4(cell);
            x[0] = f.x, x[1] = f.y, x[2] = f.z, x[3] = f.w;
          } else {
            x[0] = *cell;
          }
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            x[e] = fmaf(keep, x[e], ks[r] * v[e]);
            o[e] = fmaf(x[e], qs[r], o[e]);
          }
          if constexpr (VEC == 4) store4(cell, make_float4(x[0], x[1], x[2], x[3]));
          else *cell = x[0];
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) os[grp * width + c * VEC + e] = o[e];
      }
    }
    __syncthreads();
    float ss = 0.f;
    for (int j = threadIdx.x; j < width; j += 256) {
      float o = 0.f;
      for (int g = 0; g < groups; ++g) o += os[g * width + j];
      o *= inv_den;
      os[j] = o;
      ss += o * o;
    }
    float total = block_sum_f32(ss, red);
    if (slices > 1) {
      if (threadIdx.x == 0) s_ss[t & 1] = total;
      cluster_arrive_release();
      cluster_wait_acquire();
      total = 0.f;
      for (int i = 0; i < slices; ++i) total += ld_cluster_f32(mapa_shared(smem_u32(&s_ss[t & 1]), i));
    }
    const float inv = 1.f / sqrtf(total / static_cast<float>(dv) + p.eps);
    for (int j = threadIdx.x; j < width; j += 256) {
      const int col = h * dv + col0 + j;
      const float g = to_f32(row[2 * qk + vw + col]);
      p.out[row_i * vw + col] = from_f32<T>(os[j] * inv * p.norm_w[col] * sigmoid_f32(g));
    }
    __syncthreads();
  }
  if (slices > 1) {             // every slice has read n and m, and nobody reads a slice that has ended
    cluster_arrive_release();
    cluster_wait_acquire();
  }
  if (blockIdx.x == 0) {
    for (int i = threadIdx.x; i < dk; i += 256) n_state[i] = ns[i];
    if (threadIdx.x == 0) *m_state = m;
  }
}

constexpr int kMlstmChunkMinRows = 16;  // from this portion length on the chunk-parallel form takes over

template <typename T, int VEC>
static cudaError_t launch_mlstm_step(const MlstmParams<T>& p, int slices, cudaStream_t stream) {
  const int width = p.dv / slices, cols = width / VEC, per_row = cols < 256 ? cols : 256;
  const size_t smem = (static_cast<size_t>(3) * p.dk + static_cast<size_t>(256 / per_row) * width) * sizeof(float);
  if (smem > 48 * 1024) return cudaErrorInvalidValue;
  cudaLaunchConfig_t lc = {};
  lc.gridDim = dim3(slices, p.H, p.seqs.B);
  lc.blockDim = dim3(256);
  lc.dynamicSmemBytes = smem;
  lc.stream = stream;
  cudaLaunchAttribute attr[2];
  int n = 0;
  if (pdl_enabled()) {
    attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[n].val.programmaticStreamSerializationAllowed = 1;
    ++n;
  }
  if (slices > 1) {
    attr[n].id = cudaLaunchAttributeClusterDimension;
    attr[n].val.clusterDim.x = slices;
    attr[n].val.clusterDim.y = 1;
    attr[n].val.clusterDim.z = 1;
    ++n;
  }
  lc.attrs = attr;
  lc.numAttrs = n;
  return cudaLaunchKernelEx(&lc, mlstm_step_kernel<T, VEC>, p);
}

template <typename T>
static cudaError_t launch_mlstm_any(const MlstmParams<T>& p, int sms, cudaStream_t stream) {
  if (p.dv % 4 != 0 || p.stride % 4 != 0) return launch_mlstm_step<T, 1>(p, 1, stream);
  // enough CTAs for the machine, at least 32 columns each; beyond one per SM, slices that balance the last wave
  int slices = 1;
  auto fits = [&](int columns) { return slices < 8 && p.dv % (slices * 8) == 0 && p.dv / (slices * 2) >= columns; };
  while (fits(32) && p.H * p.seqs.B * slices < sms) slices *= 2;
  while (fits(256) && p.H * p.seqs.B * slices < 8 * sms) slices *= 2;
  return launch_mlstm_step<T, 4>(p, slices, stream);
}

}  // namespace eredu

using namespace eredu;

// Bytes of scratch a bf16 call over `rows` rows of `batch` sequences can use (0: the token-by-token kernel serves it).
extern "C" long long eredu_mlstm_scratch_bytes(int heads, int dk, int dv, int rows, int batch, int max_rows, int stride) {
  if (max_rows < kMlstmChunkMinRows || !mlstm_chunk_supported(dk, dv, 8, stride)) return 0;
  return mlstm_chunk_bytes(heads, dk, dv, rows, batch);
}

// scratch: eredu_mlstm_scratch_bytes(...) bytes of a bf16 call over `rows` rows, or null (token by token).
extern "C" int eredu_mlstm(const void* proj, const float* gates, const float* norm_w, float* state, void* out, void* scratch,
                           const int* block_table, const int* page_to_slot, const int* cu_q, const long long* slots, int heads, int dk,
                           int dv, int ld, int ldg, int stride, int rows, int batch, int q_per_seq, int max_rows, int max_pages, int fp32,
                           int sms, float cap, float eps, cudaStream_t stream) {
  if (batch <= 0 || max_rows <= 0) return 0;
  if (heads <= 0 || heads > 65535 || batch > 65535 || dk <= 0 || dv <= 0 || cap <= 0.f) return -1;
  const RaggedBatch r = {block_table, page_to_slot, cu_q, slots, batch, q_per_seq, max_pages};
  cudaError_t e;
  int launches = 1;
  if (fp32) {
    MlstmParams<float> p = {static_cast<const float*>(proj), gates, norm_w, state, static_cast<float*>(out), heads, dk, dv, ld, ldg, stride,
                            cap, eps, r};
    e = launch_mlstm_any(p, sms, stream);
  } else {
    MlstmParams<__nv_bfloat16> p = {static_cast<const __nv_bfloat16*>(proj), gates, norm_w, state, static_cast<__nv_bfloat16*>(out),
                                    heads, dk, dv, ld, ldg, stride, cap, eps, r};
    if (scratch != nullptr && max_rows >= kMlstmChunkMinRows && mlstm_chunk_supported(dk, dv, ld, stride)) {
      e = launch_mlstm_chunks(p, rows, max_rows, scratch, stream);
      launches = 3;
    } else {
      e = launch_mlstm_any(p, sms, stream);
    }
  }
  eredu_count_launches(launches);
  return static_cast<int>(e);
}
