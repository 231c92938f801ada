// Around latent attention (every head's keys and values expand from one cached vector per token):
//   * latent_prepare: RMSNorm of the query latent and of the key / value latent, rotation of the shared key part, and the append of
//     [latent | key part] as the token's cache row
//   * rotate_heads:   rotation of a slice of every query head, in place
//   * gather_rows:    cache rows into a dense matrix
//   * head_linear:    one matrix per head (queries into latent space, attended latents to values), with the rotation of a tail
//     of the input rows or a sigmoid gate on the result, and rows taken from / stored to other places
#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/launch_count.h"
#include "../common/mma.cuh"
#include "../common/ptx.cuh"

namespace eredu {

using bf16 = __nv_bfloat16;

// Sums of two values over the block in one pass; `red` holds two floats per warp.
__device__ __forceinline__ float2 block_sum2(float a, float b, float2* red) {
  a = warp_sum_f32(a);
  b = warp_sum_f32(b);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = make_float2(a, b);
  __syncthreads();
  float2 t = make_float2(0.f, 0.f);
  for (int w = 0; w < static_cast<int>(blockDim.x >> 5); ++w) {
    t.x += red[w].x;
    t.y += red[w].y;
  }
  return t;
}

// One CTA per token. proj row = [query latent (q_rank) | latent (rank) | key part (rot)]. NV > 0: rows and weights in groups of four,
// both latents fit NV groups per thread and stay in registers; NV = 0: any width and alignment.
template <typename T, int NV>
__global__ void __launch_bounds__(256) latent_prepare_kernel(const T* __restrict__ proj, T* __restrict__ cq, T* __restrict__ cache,
                                                              const int* __restrict__ positions, const long long* __restrict__ slots,
                                                              const float* __restrict__ inv_freq, const float* __restrict__ q_norm_w,
                                                              const float* __restrict__ kv_norm_w, int ld, int q_rank, int rank, int rot,
                                                              float eps) {
  __shared__ float2 red[8];
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x;
  const T* row = proj + static_cast<size_t>(m) * ld;
  const long long slot = slots[m];
  const int half = rot >> 1;
  float rot_u = 0.f, rot_v = 0.f, sn = 0.f, cs = 0.f;
  if (static_cast<int>(threadIdx.x) < half) {                        // ahead of the norms, which do not touch this part
    rot_u = to_f32(row[q_rank + rank + threadIdx.x]);
    rot_v = to_f32(row[q_rank + rank + half + threadIdx.x]);
    sincosf(static_cast<float>(positions[m]) * inv_freq[threadIdx.x], &sn, &cs);
  }
  T* q = cq + static_cast<size_t>(m) * q_rank;
  T* dst = cache + (slot >= 0 ? static_cast<size_t>(slot) * (rank + rot) : 0);
  float sq = 0.f, sk = 0.f;
  if constexpr (NV > 0) {
    const int total = q_rank + rank;
    float4 v[NV], w[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (threadIdx.x + i * 256) * 4;
      v[i] = w[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < total) {
        v[i] = load4(row + c);
        w[i] = c < q_rank ? load4(q_norm_w + c) : load4(kv_norm_w + c - q_rank);
        const float s = v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
        if (c < q_rank) sq += s;
        else sk += s;
      }
    }
    const float2 t = block_sum2(sq, sk, red);
    const float q_inv = 1.f / sqrtf(t.x / static_cast<float>(q_rank) + eps), k_inv = 1.f / sqrtf(t.y / static_cast<float>(rank) + eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (threadIdx.x + i * 256) * 4;
      if (c >= total || (c >= q_rank && slot < 0)) continue;
      const float inv = c < q_rank ? q_inv : k_inv;
      store4(c < q_rank ? q + c : dst + c - q_rank, make_float4(v[i].x * inv * w[i].x, v[i].y * inv * w[i].y, v[i].z * inv * w[i].z, v[i].w * inv * w[i].w));
    }
  } else {
    for (int c = threadIdx.x; c < q_rank; c += 256) {
      const float v = to_f32(row[c]);
      sq += v * v;
    }
    for (int c = threadIdx.x; c < rank; c += 256) {
      const float v = to_f32(row[q_rank + c]);
      sk += v * v;
    }
    const float2 t = block_sum2(sq, sk, red);
    const float q_inv = 1.f / sqrtf(t.x / static_cast<float>(q_rank) + eps), k_inv = 1.f / sqrtf(t.y / static_cast<float>(rank) + eps);
    for (int c = threadIdx.x; c < q_rank; c += 256) q[c] = from_f32<T>(to_f32(row[c]) * q_inv * q_norm_w[c]);
    if (slot >= 0)
      for (int c = threadIdx.x; c < rank; c += 256) dst[c] = from_f32<T>(to_f32(row[q_rank + c]) * k_inv * kv_norm_w[c]);
  }
  if (slot < 0) return;
  for (int i = threadIdx.x; i < half; i += 256) {
    if (i >= 256) {
      rot_u = to_f32(row[q_rank + rank + i]);
      rot_v = to_f32(row[q_rank + rank + half + i]);
      sincosf(static_cast<float>(positions[m]) * inv_freq[i], &sn, &cs);
    }
    dst[rank + i] = from_f32<T>(rot_u * cs - rot_v * sn);
    dst[rank + half + i] = from_f32<T>(rot_v * cs + rot_u * sn);
  }
}

template <typename T>
static cudaError_t launch_latent_prepare(const T* proj, T* cq, T* cache, const int* positions, const long long* slots, const float* inv_freq,
                                         const float* q_norm_w, const float* kv_norm_w, int M, int ld, int q_rank, int rank, int rot,
                                         float eps, cudaStream_t stream) {
  const uintptr_t bits = reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(cq) | reinterpret_cast<uintptr_t>(cache) |
                         reinterpret_cast<uintptr_t>(q_norm_w) | reinterpret_cast<uintptr_t>(kv_norm_w);
  const bool quads = (q_rank | rank | rot | ld) % 4 == 0 && (bits & 15) == 0;
  const int need = quads ? ((q_rank + rank) / 4 + 255) / 256 : 0;
#define ER_LP(NV_)                                                                                                                    \
  launch_pdl(latent_prepare_kernel<T, NV_>, dim3(M), dim3(256), 0, stream, proj, cq, cache, positions, slots, inv_freq, q_norm_w, kv_norm_w, ld, \
             q_rank, rank, rot, eps)
  if (need == 1) return ER_LP(1);
  if (need == 2) return ER_LP(2);
  if (need == 3 || need == 4) return ER_LP(4);
  return ER_LP(0);
#undef ER_LP
}

// x [M, heads, width]: entries [off, off + rot) of every head are turned (pairs i, i + rot / 2) by the row's position.
__global__ void __launch_bounds__(256) rotate_heads_kernel(bf16* __restrict__ x, const int* __restrict__ positions,
                                                            const float* __restrict__ inv_freq, int ld, int heads, int width, int off,
                                                            int rot) {
  extern __shared__ float cs_sn[];  // [rot / 2] cos, [rot / 2] sin
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int half = rot >> 1;
  float* cs = cs_sn;
  float* sn = cs_sn + half;
  const float pos = static_cast<float>(positions[blockIdx.x]);
  for (int i = threadIdx.x; i < half; i += 256) sincosf(pos * inv_freq[i], &sn[i], &cs[i]);
  __syncthreads();
  bf16* row = x + static_cast<size_t>(blockIdx.x) * ld + off;
  for (int i = threadIdx.x; i < heads * half; i += 256) {
    const int h = i / half, j = i - h * half;
    bf16* p = row + static_cast<size_t>(h) * width + j;
    const float u = to_f32(p[0]), v = to_f32(p[half]);
    p[0] = from_f32<bf16>(u * cs[j] - v * sn[j]);
    p[half] = from_f32<bf16>(v * cs[j] + u * sn[j]);
  }
}

// dst[i, :] = src[index[i], :], one warp per row; `pieces` 16-byte pieces (VEC) or 2-byte elements each.
template <bool VEC>
__global__ void __launch_bounds__(256) gather_rows_kernel(const uint8_t* __restrict__ src, const long long* __restrict__ index,
                                                           uint8_t* __restrict__ dst, int rows, int pieces) {
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int r = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (r >= rows) return;
  const size_t from = static_cast<size_t>(index[r]) * pieces, to = static_cast<size_t>(r) * pieces;
  if constexpr (VEC) {
    for (int c = lane; c < pieces; c += 32) reinterpret_cast<uint4*>(dst)[to + c] = reinterpret_cast<const uint4*>(src)[from + c];
  } else {
    for (int c = lane; c < pieces; c += 32) reinterpret_cast<uint16_t*>(dst)[to + c] = reinterpret_cast<const uint16_t*>(src)[from + c];
  }
}

struct HeadLinearParams {
  const void* x;         // row m, head h at x + row * ldx + h * hx
  const void* w;         // [H, N, K]
  void* out;             // row m, head h at out + row * ldy + h * hy
  const void* gate;      // row m at gate + row * ldg, column h * N + n; or null
  const int* in_rows;    // row of x (and of positions) of row m, or null: m
  const int* out_rows;   // row of out and gate of row m, or null: m
  const int* positions;  // ROT: position of every row of x
  const float* inv_freq; // ROT: [rot / 2]
  int M, H, N, K, rot;
  long long ldx, hx, ldy, hy, ldg;
};

// The tail of the input rows behind K, turned by the row's position, stored behind the N results: rows [m0, m0 + n) of head h.
template <typename T>
__device__ __forceinline__ void rotate_tail(const HeadLinearParams& p, int h, int m0, int n) {
  const int half = p.rot >> 1;
  for (int i = threadIdx.x; i < n * half; i += blockDim.x) {
    const int r = i / half, j = i - r * half;
    const int m = m0 + r;
    if (m >= p.M) break;
    const size_t src = p.in_rows != nullptr ? p.in_rows[m] : m, dst = p.out_rows != nullptr ? p.out_rows[m] : m;
    const T* x = static_cast<const T*>(p.x) + src * p.ldx + h * p.hx + p.K;
    T* y = static_cast<T*>(p.out) + dst * p.ldy + h * p.hy + p.N;
    float sn, cs;
    sincosf(static_cast<float>(p.positions[src]) * p.inv_freq[j], &sn, &cs);
    const float u = to_f32(x[j]), v = to_f32(x[half + j]);
    y[j] = from_f32<T>(u * cs - v * sn);
    y[half + j] = from_f32<T>(v * cs + u * sn);
  }
}

constexpr int kHN = 64, kHK = 64, kHStages = 3, kHStride = kHK + 8;

// grid (N tiles (+ 1 for the tail), H, M tiles), 128 threads: MT * 16 rows x 64 results, each warp 16 of the columns; K in steps of
// 64 through a cp.async ring. The head's matrix does not depend on the kernel in front, so its first tiles start before the wait.
template <int MT>
__global__ void __launch_bounds__(128) head_linear_kernel(HeadLinearParams p) {
  constexpr int ROWS = MT * 16;
  extern __shared__ __align__(16) uint8_t smem[];
  bf16* xs = reinterpret_cast<bf16*>(smem);                  // [stages][ROWS][kHStride]
  bf16* ws = xs + kHStages * ROWS * kHStride;                // [stages][64][kHStride]
  pdl_launch_early();
  const int h = blockIdx.y, m0 = blockIdx.z * ROWS, n0 = blockIdx.x * kHN;
  if (n0 >= p.N) {  // uniform: the CTA of the rotated tail
    pdl_wait();
    pdl_launch_dependents();
    rotate_tail<bf16>(p, h, m0, ROWS);
    return;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int steps = (p.K + kHK - 1) / kHK;
  const bf16* w = static_cast<const bf16*>(p.w) + static_cast<size_t>(h) * p.N * p.K;
  auto load_w = [&](int ks) {
    bf16* dst = ws + (ks % kHStages) * kHN * kHStride;
    for (int i = threadIdx.x; i < kHN * 8; i += 128) {
      const int r = i >> 3, c = (i & 7) * 8, k = ks * kHK + c;
      const bool ok = n0 + r < p.N && k < p.K;
      cp_async16(dst + r * kHStride + c, ok ? w + static_cast<size_t>(n0 + r) * p.K + k : w, ok ? 16 : 0);
    }
  };
  auto load_x = [&](int ks) {
    bf16* dst = xs + (ks % kHStages) * ROWS * kHStride;
    for (int i = threadIdx.x; i < ROWS * 8; i += 128) {
      const int r = i >> 3, c = (i & 7) * 8, k = ks * kHK + c, m = m0 + r;
      const bool ok = m < p.M && k < p.K;
      const size_t src = ok ? (p.in_rows != nullptr ? p.in_rows[m] : m) : 0;
      cp_async16(dst + r * kHStride + c, static_cast<const bf16*>(p.x) + src * p.ldx + h * p.hx + (ok ? k : 0), ok ? 16 : 0);
    }
  };
#pragma unroll
  for (int s = 0; s < kHStages - 1; ++s)
    if (s < steps) load_w(s);
  pdl_wait();
  pdl_launch_dependents();
#pragma unroll
  for (int s = 0; s < kHStages - 1; ++s) {
    if (s < steps) load_x(s);
    cp_async_commit();  // the matrix tiles issued before the wait belong to the first group
  }
  float acc[MT][2][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j) acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f;
  for (int ks = 0; ks < steps; ++ks) {
    cp_async_wait<kHStages - 2>();
    __syncthreads();
    if (ks + kHStages - 1 < steps) {
      load_w(ks + kHStages - 1);
      load_x(ks + kHStages - 1);
    }
    cp_async_commit();
    const bf16* xt = xs + (ks % kHStages) * ROWS * kHStride;
    const bf16* wt = ws + (ks % kHStages) * kHN * kHStride;
#pragma unroll
    for (int kk = 0; kk < kHK / 16; ++kk) {
      uint32_t b0, b1, b2, b3;
      ldsm_x4(smem_u32(wt + (warp * 16 + (lane & 7) + (lane >> 4) * 8) * kHStride + kk * 16 + ((lane >> 3) & 1) * 8), b0, b1, b2, b3);
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        uint32_t a0, a1, a2, a3;
        ldsm_x4(smem_u32(xt + (i * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kHStride + kk * 16 + (lane >> 4) * 8), a0, a1, a2, a3);
        mma16816(acc[i][0], a0, a1, a2, a3, b0, b1);
        mma16816(acc[i][1], a0, a1, a2, a3, b2, b3);
      }
    }
  }
  const int g = lane >> 2, tig = lane & 3;
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int m = m0 + i * 16 + g + r * 8;
      if (m >= p.M) continue;
      const size_t dst = p.out_rows != nullptr ? p.out_rows[m] : m;
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int n = n0 + warp * 16 + j * 8 + tig * 2;
        if (n >= p.N) continue;
        float a = acc[i][j][2 * r], b = acc[i][j][2 * r + 1];
        if (p.gate != nullptr) {
          const uint32_t gt = *reinterpret_cast<const uint32_t*>(static_cast<const bf16*>(p.gate) + dst * p.ldg + static_cast<size_t>(h) * p.N + n);
          a *= sigmoid_fast(bf16_lo(gt));
          b *= sigmoid_fast(bf16_hi(gt));
        }
        *reinterpret_cast<uint32_t*>(static_cast<bf16*>(p.out) + dst * p.ldy + h * p.hy + n) = pack_bf16x2(a, b);
      }
    }
}

// Any sizes and pitches, fp32 or bf16, fp32 arithmetic: 16 rows x 16 results per CTA through shared memory.
template <typename T>
__global__ void __launch_bounds__(256) head_linear_simt_kernel(HeadLinearParams p) {
  __shared__ float xs[16][17], ws[16][17];
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int h = blockIdx.y, m0 = blockIdx.z * 16, n0 = blockIdx.x * 16;
  if (n0 >= p.N) {
    rotate_tail<T>(p, h, m0, 16);
    return;
  }
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const T* w = static_cast<const T*>(p.w) + static_cast<size_t>(h) * p.N * p.K;
  const int ml = m0 + ty;
  const size_t src = ml < p.M ? (p.in_rows != nullptr ? p.in_rows[ml] : ml) : 0;
  const T* x = static_cast<const T*>(p.x) + src * p.ldx + h * p.hx;
  float acc = 0.f;
  for (int k0 = 0; k0 < p.K; k0 += 16) {
    xs[ty][tx] = ml < p.M && k0 + tx < p.K ? to_f32(x[k0 + tx]) : 0.f;
    ws[ty][tx] = n0 + ty < p.N && k0 + tx < p.K ? to_f32(w[static_cast<size_t>(n0 + ty) * p.K + k0 + tx]) : 0.f;
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) acc = fmaf(xs[ty][k], ws[tx][k], acc);
    __syncthreads();
  }
  const int n = n0 + tx;
  if (ml >= p.M || n >= p.N) return;
  const size_t dst = p.out_rows != nullptr ? p.out_rows[ml] : ml;
  if (p.gate != nullptr) acc *= sigmoid_f32(to_f32(static_cast<const T*>(p.gate)[dst * p.ldg + static_cast<size_t>(h) * p.N + n]));
  static_cast<T*>(p.out)[dst * p.ldy + h * p.hy + n] = from_f32<T>(acc);
}

template <int MT>
static cudaError_t launch_head_linear(const HeadLinearParams& p, cudaStream_t stream) {
  constexpr size_t smem = kHStages * (MT * 16 + kHN) * kHStride * sizeof(bf16);
  static bool configured[64] = {};
  int dev = 0;
  cudaError_t e = cudaGetDevice(&dev);
  if (e != cudaSuccess) return e;
  if (dev < 0 || dev >= 64) return cudaErrorInvalidDevice;
  if (!configured[dev]) {
    e = cudaFuncSetAttribute(head_linear_kernel<MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return e;
    configured[dev] = true;
  }
  const dim3 grid((p.N + kHN - 1) / kHN + (p.rot > 0 ? 1 : 0), p.H, (p.M + MT * 16 - 1) / (MT * 16));
  if (grid.z > 65535) return cudaErrorInvalidValue;
  return launch_pdl(head_linear_kernel<MT>, grid, dim3(128), smem, stream, p);
}

}  // namespace eredu

using namespace eredu;

extern "C" int eredu_latent_prepare(const void* proj, void* cq, void* cache, const int* positions, const long long* slots,
                                    const float* inv_freq, const float* q_norm_w, const float* kv_norm_w, int M, int ld, int q_rank,
                                    int rank, int rot, int fp32, float eps, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (q_rank <= 0 || rank <= 0 || rot < 0 || rot % 2 != 0) return -1;
  const cudaError_t e =
      fp32 ? launch_latent_prepare(static_cast<const float*>(proj), static_cast<float*>(cq), static_cast<float*>(cache), positions, slots, inv_freq,
                                   q_norm_w, kv_norm_w, M, ld, q_rank, rank, rot, eps, stream)
           : launch_latent_prepare(static_cast<const bf16*>(proj), static_cast<bf16*>(cq), static_cast<bf16*>(cache), positions, slots, inv_freq,
                                   q_norm_w, kv_norm_w, M, ld, q_rank, rank, rot, eps, stream);
  eredu_count_launches(1);
  return static_cast<int>(e);
}

extern "C" int eredu_rotate_heads(void* x, const int* positions, const float* inv_freq, int M, int ld, int heads, int width, int off,
                                  int rot, cudaStream_t stream) {
  if (M <= 0 || rot <= 0) return 0;
  if (rot % 2 != 0 || off < 0 || off + rot > width || rot > 4096) return -1;
  const cudaError_t e = launch_pdl(rotate_heads_kernel, dim3(M), dim3(256), rot * sizeof(float), stream, static_cast<bf16*>(x), positions,
                                   inv_freq, ld, heads, width, off, rot);
  eredu_count_launches(1);
  return static_cast<int>(e);
}

// dst [rows, width] = src rows `index`; elements of 2 or 4 bytes.
extern "C" int eredu_gather_rows(const void* src, const long long* index, void* dst, int rows, int width, int elem_bytes,
                                 cudaStream_t stream) {
  if (rows <= 0 || width <= 0) return 0;
  if (elem_bytes != 2 && elem_bytes != 4) return -1;
  const int bytes = width * elem_bytes;
  const bool vec = bytes % 16 == 0 && ((reinterpret_cast<uintptr_t>(src) | reinterpret_cast<uintptr_t>(dst)) & 15) == 0;
  const dim3 grid((rows + 7) / 8);
  const uint8_t* s = static_cast<const uint8_t*>(src);
  uint8_t* d = static_cast<uint8_t*>(dst);
  const cudaError_t e = vec ? launch_pdl(gather_rows_kernel<true>, grid, dim3(256), 0, stream, s, index, d, rows, bytes / 16)
                            : launch_pdl(gather_rows_kernel<false>, grid, dim3(256), 0, stream, s, index, d, rows, bytes / 2);
  eredu_count_launches(1);
  return static_cast<int>(e);
}

// tc: all sizes and pitches are multiples of 8 elements and the pointers are aligned (tensor-core form, bf16).
extern "C" int eredu_head_linear(const void* x, const void* w, void* out, const void* gate, const int* in_rows, const int* out_rows,
                                 const int* positions, const float* inv_freq, int M, int H, int N, int K, long long ldx, long long hx,
                                 long long ldy, long long hy, long long ldg, int rot, int fp32, int tc, cudaStream_t stream) {
  if (M <= 0 || H <= 0 || N <= 0) return 0;
  if (K <= 0 || rot < 0 || rot % 2 != 0 || H > 65535 || (rot > 0 && (positions == nullptr || inv_freq == nullptr))) return -1;
  HeadLinearParams p = {x, w, out, gate, in_rows, out_rows, positions, inv_freq, M, H, N, K, rot, ldx, hx, ldy, hy, ldg};
  cudaError_t e;
  if (tc && !fp32) {
    e = M <= 16 ? launch_head_linear<1>(p, stream) : M <= 32 ? launch_head_linear<2>(p, stream) : launch_head_linear<4>(p, stream);
  } else {
    const dim3 grid((N + 15) / 16 + (rot > 0 ? 1 : 0), H, (M + 15) / 16);
    if (grid.z > 65535) return -1;
    e = fp32 ? launch_pdl(head_linear_simt_kernel<float>, grid, dim3(256), 0, stream, p)
             : launch_pdl(head_linear_simt_kernel<bf16>, grid, dim3(256), 0, stream, p);
  }
  eredu_count_launches(1);
  return static_cast<int>(e);
}
