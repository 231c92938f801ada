// Glue of decoders that keep their residual stream in fp32:
//   * residual_norm: x' = x + y + the weighted expert rows of the token, and LayerNorm or RMSNorm of x' for the next layer
//   * rms_residual (a norm on a sublayer's OUTPUT): x = residual + w * y / rms(y), in fp32, plus the copy of x in the compute dtype that the next
//     projections read (one number or one vector as w; without a residual: a plain norm, as in front of the head)
//   * branch_norm (norms in front of and behind a sublayer): x' = x + w rms(gain (y0 + y1)), the branches normed by themselves first
//     where they have weights, and the norm of x' in front of the next sublayer
//   * rms_routed_residual: rms_residual of a sublayer's output plus weighted expert rows; the copy may be x + conv(x) in decode steps
//   * stream_conv: x + conv(x), a causal convolution over the stream with the last inputs as state
//   * embedding_stream: the first rows of the stream and their copy, with sinusoidal position vectors where a model adds them
//   * qkv_prepare: RMSNorm over the WHOLE query and key projections, rotation of the leading dims of every head, RMSNorm of
//     every value head, and the append to the paged cache, whose key and value widths may differ
// All of them for bf16 and for fp32 activations.
#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/launch_count.h"
#include "../common/ptx.cuh"
#include "../common/ragged.cuh"

namespace eredu {

// One CTA per row; NV groups of four columns per thread stay in registers between the two passes. NV = 0: any width, the
// row is read twice.
template <typename TY, int NV>
__global__ void __launch_bounds__(256) rms_residual_kernel(const TY* __restrict__ y, const float* __restrict__ w, int w_vec,
                                                            const float* __restrict__ residual, float* __restrict__ x_out,
                                                            __nv_bfloat16* __restrict__ act, int W, float eps) {
  __shared__ float red[8];
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const size_t base = static_cast<size_t>(blockIdx.x) * W;
  const float w0 = w[0];
  if constexpr (NV > 0) {
    float4 v[NV], rv[NV];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (threadIdx.x + i * 256) * 4;
      v[i] = rv[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < W) {
        v[i] = load4(y + base + c);
        if (residual != nullptr) rv[i] = load4(residual + base + c);
      }
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    const float inv = 1.f / sqrtf(block_sum_f32(ss, red) / static_cast<float>(W) + eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (threadIdx.x + i * 256) * 4;
      if (c >= W) continue;
      const float4 g = w_vec ? load4(w + c) : make_float4(w0, w0, w0, w0);
      const float4 o = make_float4(rv[i].x + v[i].x * inv * g.x, rv[i].y + v[i].y * inv * g.y, rv[i].z + v[i].z * inv * g.z,
                                   rv[i].w + v[i].w * inv * g.w);
      if (x_out != nullptr) store4(x_out + base + c, o);
      if (act != nullptr) store4(act + base + c, o);
    }
  } else {
    float ss = 0.f;
    for (int c = threadIdx.x; c < W; c += 256) {
      const float t = to_f32(y[base + c]);
      ss += t * t;
    }
    const float inv = 1.f / sqrtf(block_sum_f32(ss, red) / static_cast<float>(W) + eps);
    for (int c = threadIdx.x; c < W; c += 256) {
      const float o = (residual != nullptr ? residual[base + c] : 0.f) + to_f32(y[base + c]) * inv * (w_vec ? w[c] : w0);
      if (x_out != nullptr) x_out[base + c] = o;
      if (act != nullptr) act[base + c] = __float2bfloat16(o);
    }
  }
}

template <typename TY>
static cudaError_t launch_rms_residual(const TY* y, const float* w, int w_vec, const float* residual, float* x_out, __nv_bfloat16* act,
                                       int M, int W, float eps, cudaStream_t stream) {
  const int quads = W % 4 == 0 ? (W / 4 + 255) / 256 : 0;
#define ER_RMS(NV_) launch_pdl(rms_residual_kernel<TY, NV_>, dim3(M), dim3(256), 0, stream, y, w, w_vec, residual, x_out, act, W, eps)
  switch (quads) {
    case 1: return ER_RMS(1);
    case 2: return ER_RMS(2);
    case 3:
    case 4: return ER_RMS(4);
    case 5:
    case 6:
    case 7:
    case 8: return ER_RMS(8);
    default: return ER_RMS(0);
  }
#undef ER_RMS
}

struct ResidualNormParams {
  const float* x;           // [M, W]
  const void* y;            // [M, W] a sublayer's output, or null
  const void* rows;         // expert outputs, or null
  const int* route_pos;     // [M * k] row of a route, negative: none
  const float* route_w;     // [M * k]
  const float* weight;      // [W], or null: no norm
  const float* bias;        // [W] or null
  float* x_out;             // [M, W]; null when nothing is added
  void* act;                // [M, W]
  int W, k, center;
  float eps;
};

constexpr int kMaxRoutes = 32;

// One CTA per row. NV groups of four columns per thread stay in registers; NV = 0: any width, the sum is read back.
template <typename T, int NV>
__global__ void __launch_bounds__(256) residual_norm_kernel(ResidualNormParams p) {
  __shared__ float red[8];
  __shared__ int pos[kMaxRoutes];
  __shared__ float rw[kMaxRoutes];
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int W = p.W;
  const size_t base = static_cast<size_t>(blockIdx.x) * W;
  const T* y = static_cast<const T*>(p.y);
  const T* rows = static_cast<const T*>(p.rows);
  T* act = static_cast<T*>(p.act);
  const float n = static_cast<float>(W);
  if (p.k > 0) {
    if (threadIdx.x < p.k) {
      pos[threadIdx.x] = p.route_pos[static_cast<size_t>(blockIdx.x) * p.k + threadIdx.x];
      rw[threadIdx.x] = p.route_w[static_cast<size_t>(blockIdx.x) * p.k + threadIdx.x];
    }
    __syncthreads();
  }
  if constexpr (NV > 0) {
    float4 v[NV];
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (threadIdx.x + i * 256) * 4;
      v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < W) {
        v[i] = load4(p.x + base + c);
        if (y != nullptr) {
          const float4 a = load4(y + base + c);
          v[i] = make_float4(v[i].x + a.x, v[i].y + a.y, v[i].z + a.z, v[i].w + a.w);
        }
      }
    }
#pragma unroll 4
    for (int s = 0; s < p.k; ++s) {
      if (pos[s] < 0) continue;
      const T* r = rows + static_cast<size_t>(pos[s]) * W;
      const float w = rw[s];
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = (threadIdx.x + i * 256) * 4;
        if (c >= W) continue;
        const float4 a = load4(r + c);
        v[i] = make_float4(fmaf(w, a.x, v[i].x), fmaf(w, a.y, v[i].y), fmaf(w, a.z, v[i].z), fmaf(w, a.w, v[i].w));
      }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (threadIdx.x + i * 256) * 4;
      if (c < W && p.x_out != nullptr) store4(p.x_out + base + c, v[i]);
      sum += v[i].x + v[i].y + v[i].z + v[i].w;
    }
    if (p.weight == nullptr) return;
    const float mean = p.center ? block_sum_f32(sum, red) / n : 0.f;
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      if ((threadIdx.x + i * 256) * 4 >= W) continue;
      v[i] = make_float4(v[i].x - mean, v[i].y - mean, v[i].z - mean, v[i].w - mean);
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    const float inv = 1.f / sqrtf(block_sum_f32(ss, red) / n + p.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (threadIdx.x + i * 256) * 4;
      if (c >= W) continue;
      const float4 g = load4(p.weight + c);
      const float4 b = p.bias != nullptr ? load4(p.bias + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      store4(act + base + c, make_float4(fmaf(v[i].x * inv, g.x, b.x), fmaf(v[i].y * inv, g.y, b.y), fmaf(v[i].z * inv, g.z, b.z),
                                         fmaf(v[i].w * inv, g.w, b.w)));
    }
  } else {
    const float* src = p.x_out != nullptr ? p.x_out : p.x;      // a thread reads back only what it wrote itself
    float sum = 0.f;
    for (int c = threadIdx.x; c < W; c += 256) {
      float v = p.x[base + c];
      if (y != nullptr) v += to_f32(y[base + c]);
      for (int s = 0; s < p.k; ++s)
        if (pos[s] >= 0) v = fmaf(rw[s], to_f32(rows[static_cast<size_t>(pos[s]) * W + c]), v);
      if (p.x_out != nullptr) p.x_out[base + c] = v;
      sum += v;
    }
    if (p.weight == nullptr) return;
    const float mean = p.center ? block_sum_f32(sum, red) / n : 0.f;
    float ss = 0.f;
    for (int c = threadIdx.x; c < W; c += 256) {
      const float d = src[base + c] - mean;
      ss += d * d;
    }
    const float inv = 1.f / sqrtf(block_sum_f32(ss, red) / n + p.eps);
    for (int c = threadIdx.x; c < W; c += 256)
      act[base + c] = from_f32<T>(fmaf((src[base + c] - mean) * inv, p.weight[c], p.bias != nullptr ? p.bias[c] : 0.f));
  }
}

template <typename T>
static cudaError_t launch_residual_norm(const ResidualNormParams& p, int M, bool quads_ok, cudaStream_t stream) {
  const int quads = quads_ok ? (p.W / 4 + 255) / 256 : 0;
#define ER_RN(NV_) launch_pdl(residual_norm_kernel<T, NV_>, dim3(M), dim3(256), 0, stream, p)
  switch (quads) {
    case 1: return ER_RN(1);
    case 2: return ER_RN(2);
    case 3:
    case 4: return ER_RN(4);
    case 5:
    case 6:
    case 7:
    case 8: return ER_RN(8);
    default: return ER_RN(0);
  }
#undef ER_RN
}

struct BranchNormParams {
  const float* x;           // [M, W]
  const void* y0;           // [M, W]
  const void* y1;           // [M, W] or null
  const float* w0;          // [W] norms of the branches, or null
  const float* w1;
  const float* weight;      // [W] norm of their sum
  const float* next;        // [W] or null: no activations
  float* x_out;
  void* act;
  int W;
  float gain, eps;
};

// Sums over a block of 256 threads with one barrier; `red` is not used again.
__device__ __forceinline__ float block_sum_once(float v, float* red) {
  v = warp_sum_f32(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  const float4 a = load4(red), b = load4(red + 4);
  return ((a.x + a.y) + (a.z + a.w)) + ((b.x + b.y) + (b.z + b.w));
}
__device__ __forceinline__ float2 block_sum2_once(float u, float v, float* red) {
  u = warp_sum_f32(u);
  v = warp_sum_f32(v);
  if ((threadIdx.x & 31) == 0) {
    red[threadIdx.x >> 5] = u;
    red[8 + (threadIdx.x >> 5)] = v;
  }
  __syncthreads();
  const float4 a = load4(red), b = load4(red + 4), c = load4(red + 8), d = load4(red + 12);
  return make_float2(((a.x + a.y) + (a.z + a.w)) + ((b.x + b.y) + (b.z + b.w)), ((c.x + c.y) + (c.z + c.w)) + ((d.x + d.y) + (d.z + d.w)));
}

// x' = x + rms(gain (y0 + y1)) weight (each branch RMS-normed by itself first where it has a weight), act = rms(x') next. One CTA per row;
// NV groups of four columns per thread stay in registers; NV = 0: any width, rows are read again.
template <typename T, int NV>
__global__ void __launch_bounds__(256) branch_norm_kernel(BranchNormParams p) {
  __shared__ __align__(16) float red2[16], red_y[8], red_x[8];
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int W = p.W;
  const size_t base = static_cast<size_t>(blockIdx.x) * W;
  const T* y0 = static_cast<const T*>(p.y0) + base;
  const T* y1 = p.y1 != nullptr ? static_cast<const T*>(p.y1) + base : nullptr;
  T* act = static_cast<T*>(p.act);
  const float n = static_cast<float>(W);
  float i0 = 1.f, i1 = 1.f;
  if constexpr (NV > 0) {
    float4 v[NV], x[NV];
    {
      float4 u[NV];
      float s0 = 0.f, s1 = 0.f;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = (threadIdx.x + i * 256) * 4;
        v[i] = u[i] = x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < W) {
          v[i] = load4(y0 + c);
          if (y1 != nullptr) u[i] = load4(y1 + c);
          x[i] = load4(p.x + base + c);
        }
        s0 += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
        s1 += u[i].x * u[i].x + u[i].y * u[i].y + u[i].z * u[i].z + u[i].w * u[i].w;
      }
      if (p.w0 != nullptr) {
        const float2 t = block_sum2_once(s0, s1, red2);
        i0 = 1.f / sqrtf(t.x / n + p.eps);
        i1 = 1.f / sqrtf(t.y / n + p.eps);
      }
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = (threadIdx.x + i * 256) * 4;
        if (c >= W) continue;
        float4 a = make_float4(i0, i0, i0, i0), b = make_float4(i1, i1, i1, i1);
        if (p.w0 != nullptr) {
          const float4 g = load4(p.w0 + c);
          a = make_float4(a.x * g.x, a.y * g.y, a.z * g.z, a.w * g.w);
        }
        if (p.w1 != nullptr) {
          const float4 g = load4(p.w1 + c);
          b = make_float4(b.x * g.x, b.y * g.y, b.z * g.z, b.w * g.w);
        }
        v[i] = make_float4(p.gain * fmaf(v[i].x, a.x, u[i].x * b.x), p.gain * fmaf(v[i].y, a.y, u[i].y * b.y), p.gain * fmaf(v[i].z, a.z, u[i].z * b.z),
                           p.gain * fmaf(v[i].w, a.w, u[i].w * b.w));
      }
    }
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    const float inv = 1.f / sqrtf(block_sum_once(ss, red_y) / n + p.eps);
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (threadIdx.x + i * 256) * 4;
      if (c >= W) continue;
      const float4 g = load4(p.weight + c);
      x[i] = make_float4(fmaf(v[i].x * inv, g.x, x[i].x), fmaf(v[i].y * inv, g.y, x[i].y), fmaf(v[i].z * inv, g.z, x[i].z), fmaf(v[i].w * inv, g.w, x[i].w));
      store4(p.x_out + base + c, x[i]);
      ss += x[i].x * x[i].x + x[i].y * x[i].y + x[i].z * x[i].z + x[i].w * x[i].w;
    }
    if (p.next == nullptr) return;
    const float out = 1.f / sqrtf(block_sum_once(ss, red_x) / n + p.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (threadIdx.x + i * 256) * 4;
      if (c >= W) continue;
      const float4 g = load4(p.next + c);
      store4(act + base + c, make_float4(x[i].x * out * g.x, x[i].y * out * g.y, x[i].z * out * g.z, x[i].w * out * g.w));
    }
  } else {
    if (p.w0 != nullptr) {
      float s0 = 0.f, s1 = 0.f;
      for (int c = threadIdx.x; c < W; c += 256) {
        const float a = to_f32(y0[c]), b = y1 != nullptr ? to_f32(y1[c]) : 0.f;
        s0 += a * a;
        s1 += b * b;
      }
      const float2 t = block_sum2_once(s0, s1, red2);
      i0 = 1.f / sqrtf(t.x / n + p.eps);
      i1 = 1.f / sqrtf(t.y / n + p.eps);
    }
    auto mixed = [&](int c) {
      const float a = to_f32(y0[c]) * i0 * (p.w0 != nullptr ? p.w0[c] : 1.f);
      const float b = y1 != nullptr ? to_f32(y1[c]) * i1 * (p.w1 != nullptr ? p.w1[c] : 1.f) : 0.f;
      return p.gain * (a + b);
    };
    float ss = 0.f;
    for (int c = threadIdx.x; c < W; c += 256) {
      const float m = mixed(c);
      ss += m * m;
    }
    const float inv = 1.f / sqrtf(block_sum_once(ss, red_y) / n + p.eps);
    ss = 0.f;
    for (int c = threadIdx.x; c < W; c += 256) {
      const float o = fmaf(mixed(c) * inv, p.weight[c], p.x[base + c]);
      p.x_out[base + c] = o;
      ss += o * o;
    }
    if (p.next == nullptr) return;
    const float out = 1.f / sqrtf(block_sum_once(ss, red_x) / n + p.eps);
    for (int c = threadIdx.x; c < W; c += 256) act[base + c] = from_f32<T>(p.x_out[base + c] * out * p.next[c]);
  }
}

template <typename T>
static cudaError_t launch_branch_norm(const BranchNormParams& p, int M, bool quads_ok, cudaStream_t stream) {
  const int quads = quads_ok ? (p.W / 4 + 255) / 256 : 0;
#define ER_BN(NV_) launch_pdl(branch_norm_kernel<T, NV_>, dim3(M), dim3(256), 0, stream, p)
  switch (quads) {
    case 1: return ER_BN(1);
    case 2: return ER_BN(2);
    case 3:
    case 4: return ER_BN(4);
    case 5:
    case 6:
    case 7:
    case 8: return ER_BN(8);
    default: return ER_BN(0);
  }
#undef ER_BN
}

struct RoutedResidualParams {
  const void* y;            // [M, W] a sublayer's output, or null
  const void* rows;         // expert outputs, or null
  const int* route_pos;     // [M * k] row of a route, negative: none
  const float* route_w;     // [M * k]
  const float* weight;      // [W]
  const float* residual;    // [M, W]
  float* x_out;             // [M, W]
  void* act;                // [M, W] or null
  // decode steps of one row per sequence: act = x' + conv(x')
  const float* taps;        // [taps, W] or null
  float* state;             // [slots, state_elems] of which the first (taps - 1) W are the last inputs, oldest first; null: one tap
  RaggedBatch seqs;
  int n_taps, state_elems;
  int W, k;
  float eps;
};

// One CTA per row: x' = residual + weight rms(y + sum_k w_k rows_k). NV groups of four columns per thread stay in registers; NV = 0: any
// width, the sum is formed twice. CONV: with the convolution.
template <typename T, int NV, bool CONV>
__global__ void __launch_bounds__(256) rms_routed_residual_kernel(RoutedResidualParams p) {
  __shared__ __align__(16) float red[8];
  __shared__ int pos[kMaxRoutes];
  __shared__ float rw[kMaxRoutes];
  pdl_launch_early();
  const int W = p.W;
  pdl_wait();
  pdl_launch_dependents();
  const size_t base = static_cast<size_t>(blockIdx.x) * W;
  const T* y = p.y != nullptr ? static_cast<const T*>(p.y) + base : nullptr;
  const T* rows = static_cast<const T*>(p.rows);
  T* act = p.act != nullptr ? static_cast<T*>(p.act) + base : nullptr;
  if (p.k > 0) {
    if (threadIdx.x < p.k) {
      pos[threadIdx.x] = p.route_pos[static_cast<size_t>(blockIdx.x) * p.k + threadIdx.x];
      rw[threadIdx.x] = p.route_w[static_cast<size_t>(blockIdx.x) * p.k + threadIdx.x];
    }
    __syncthreads();
  }
  float* hist = nullptr;
  if (p.state != nullptr) {
    const RaggedSeq s = ragged_seq(p.seqs, blockIdx.x);
    if (s.live) hist = p.state + static_cast<size_t>(s.slot) * p.state_elems;
  }
  const float n = static_cast<float>(W);
  if constexpr (NV > 0) {
    float4 v[NV], rv[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (threadIdx.x + i * 256) * 4;
      v[i] = rv[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < W) {
        if (y != nullptr) v[i] = load4(y + c);
        rv[i] = load4(p.residual + base + c);
      }
    }
#pragma unroll 4
    for (int s = 0; s < p.k; ++s) {
      if (pos[s] < 0) continue;
      const T* r = rows + static_cast<size_t>(pos[s]) * W;
      const float w = rw[s];
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = (threadIdx.x + i * 256) * 4;
        if (c >= W) continue;
        const float4 a = load4(r + c);
        v[i] = make_float4(fmaf(w, a.x, v[i].x), fmaf(w, a.y, v[i].y), fmaf(w, a.z, v[i].z), fmaf(w, a.w, v[i].w));
      }
    }
    // the first rows of the history travel while the sum is formed
    constexpr int AHEAD = CONV && NV <= 4 ? 3 : 0;
    float4 past[NV][AHEAD > 0 ? AHEAD : 1];
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
      for (int j = 0; j < AHEAD; ++j) {
        const int c = (threadIdx.x + i * 256) * 4;
        if (hist != nullptr && c < W && j < p.n_taps - 1) past[i][j] = load4(hist + static_cast<size_t>(j) * W + c);
      }
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    const float inv = 1.f / sqrtf(block_sum_once(ss, red) / n + p.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (threadIdx.x + i * 256) * 4;
      if (c >= W) continue;
      const float4 g = load4(p.weight + c);
      const float4 o = make_float4(fmaf(v[i].x * inv, g.x, rv[i].x), fmaf(v[i].y * inv, g.y, rv[i].y), fmaf(v[i].z * inv, g.z, rv[i].z),
                                   fmaf(v[i].w * inv, g.w, rv[i].w));
      store4(p.x_out + base + c, o);
      if (act == nullptr) continue;
      float4 h = o;
      if constexpr (CONV) {
        auto tap = [&](int j, const float4& u) {
          const float4 t = load4(p.taps + static_cast<size_t>(j) * W + c);
          if (j > 0 && hist != nullptr) store4(hist + static_cast<size_t>(j - 1) * W + c, u);
          h = make_float4(fmaf(t.x, u.x, h.x), fmaf(t.y, u.y, h.y), fmaf(t.z, u.z, h.z), fmaf(t.w, u.w, h.w));
        };
        if (hist != nullptr) {
#pragma unroll
          for (int j = 0; j < AHEAD; ++j)
            if (j < p.n_taps - 1) tap(j, past[i][j]);
          for (int j = AHEAD; j < p.n_taps - 1; ++j) tap(j, load4(hist + static_cast<size_t>(j) * W + c));
        }
        tap(p.n_taps - 1, o);
      }
      store4(act + c, h);
    }
  } else {
    auto summed = [&](int c) {
      float t = y != nullptr ? to_f32(y[c]) : 0.f;
      for (int s = 0; s < p.k; ++s)
        if (pos[s] >= 0) t = fmaf(rw[s], to_f32(rows[static_cast<size_t>(pos[s]) * W + c]), t);
      return t;
    };
    float ss = 0.f;
    for (int c = threadIdx.x; c < W; c += 256) {
      const float t = summed(c);
      ss += t * t;
    }
    const float inv = 1.f / sqrtf(block_sum_once(ss, red) / n + p.eps);
    for (int c = threadIdx.x; c < W; c += 256) {
      const float o = fmaf(summed(c) * inv, p.weight[c], p.residual[base + c]);
      p.x_out[base + c] = o;
      if (act == nullptr) continue;
      float h = o;
      if constexpr (CONV) {
        for (int j = 0; j < p.n_taps; ++j) {
          const bool own = j == p.n_taps - 1;
          if (!own && hist == nullptr) continue;
          const float u = own ? o : hist[static_cast<size_t>(j) * W + c];
          if (j > 0 && hist != nullptr) hist[static_cast<size_t>(j - 1) * W + c] = u;
          h = fmaf(p.taps[static_cast<size_t>(j) * W + c], u, h);
        }
      }
      act[c] = from_f32<T>(h);
    }
  }
}

template <typename T>
static cudaError_t launch_rms_routed_residual(const RoutedResidualParams& p, int M, bool quads_ok, cudaStream_t stream) {
  const int quads = quads_ok ? (p.W / 4 + 255) / 256 : 0;
#define ER_RR(NV_) \
  (p.taps != nullptr ? launch_pdl(rms_routed_residual_kernel<T, NV_, true>, dim3(M), dim3(256), 0, stream, p) \
                     : launch_pdl(rms_routed_residual_kernel<T, NV_, false>, dim3(M), dim3(256), 0, stream, p))
  switch (quads) {
    case 1: return ER_RR(1);
    case 2: return ER_RR(2);
    case 3:
    case 4: return ER_RR(4);
    case 5:
    case 6:
    case 7:
    case 8: return ER_RR(8);
    default: return ER_RR(0);
  }
#undef ER_RR
}

struct StreamConvParams {
  const float* x;       // [M, W]
  void* act;            // [M, W]
  const float* taps;    // [taps, W]
  float* state;         // as RoutedResidualParams
  RaggedBatch seqs;
  int W, n_taps, state_elems, tile;   // tile: rows of a CTA, at least taps - 1
};

template <int VEC>
__device__ __forceinline__ void load_vec(float (&v)[VEC], const float* p) {
  if constexpr (VEC == 4) {
    const float4 f = load4(p);
    v[0] = f.x;
    v[1] = f.y;
    v[2] = f.z;
    v[3] = f.w;
  } else {
    v[0] = *p;
  }
}
template <int VEC, typename T>
__device__ __forceinline__ void store_vec(T* p, const float (&v)[VEC]) {
  if constexpr (VEC == 4) store4(p, make_float4(v[0], v[1], v[2], v[3]));
  else *p = from_f32<T>(v[0]);
}

// A thread owns VEC channels of one tile of a sequence's rows. L > 0: that many taps, the last inputs in registers; L = 0: any number,
// inputs are read again. The thread that has the sequence's first rows also moves the history on, after it has read it.
template <typename T, int VEC, int L>
__global__ void __launch_bounds__(256) stream_conv_kernel(StreamConvParams p) {
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int W = p.W, c = (blockIdx.x * 256 + threadIdx.x) * VEC;
  const RaggedSeq s = ragged_seq(p.seqs, blockIdx.z);
  const int t0 = blockIdx.y * p.tile, t1 = min(t0 + p.tile, s.rows), n_taps = L > 0 ? L : p.n_taps;
  if (t0 >= s.rows || c >= W) return;
  const float* x = p.x + static_cast<size_t>(s.row0) * W + c;
  T* act = static_cast<T*>(p.act) + static_cast<size_t>(s.row0) * W + c;
  float* hist = p.state != nullptr && s.live ? p.state + static_cast<size_t>(s.slot) * p.state_elems + c : nullptr;
  // input of position t of this portion, t >= -(taps - 1)
  auto input = [&](float (&v)[VEC], int t) {
    if (t >= 0) load_vec<VEC>(v, x + static_cast<size_t>(t) * W);
    else if (hist != nullptr) load_vec<VEC>(v, hist + static_cast<size_t>(t + n_taps - 1) * W);
    else
      for (int e = 0; e < VEC; ++e) v[e] = 0.f;
  };
  if constexpr (L > 0) {
    float w[L][VEC], in[L][VEC];
#pragma unroll
    for (int j = 0; j < L; ++j) load_vec<VEC>(w[j], p.taps + static_cast<size_t>(j) * W + c);
#pragma unroll
    for (int j = 0; j + 1 < L; ++j) input(in[j + 1], t0 - (L - 1) + j);
#pragma unroll 4
    for (int t = t0; t < t1; ++t) {
#pragma unroll
      for (int j = 0; j + 1 < L; ++j)
#pragma unroll
        for (int e = 0; e < VEC; ++e) in[j][e] = in[j + 1][e];
      load_vec<VEC>(in[L - 1], x + static_cast<size_t>(t) * W);
      float h[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        h[e] = in[L - 1][e];
#pragma unroll
        for (int j = 0; j < L; ++j) h[e] = fmaf(w[j][e], in[j][e], h[e]);
      }
      store_vec<VEC>(act + static_cast<size_t>(t) * W, h);
    }
  } else {
    for (int t = t0; t < t1; ++t) {
      float h[VEC], u[VEC], w[VEC];
      load_vec<VEC>(h, x + static_cast<size_t>(t) * W);
      for (int j = 0; j < n_taps; ++j) {
        input(u, t - (n_taps - 1) + j);
        load_vec<VEC>(w, p.taps + static_cast<size_t>(j) * W + c);
#pragma unroll
        for (int e = 0; e < VEC; ++e) h[e] = fmaf(w[e], u[e], h[e]);
      }
      store_vec<VEC>(act + static_cast<size_t>(t) * W, h);
    }
  }
  if (t0 > 0 || hist == nullptr) return;
  for (int j = 0; j + 1 < n_taps; ++j) {      // what row j takes lies behind it: upwards, in place
    float v[VEC];
    input(v, s.rows - (n_taps - 1) + j);
    store_vec<VEC>(hist + static_cast<size_t>(j) * W, v);
  }
}

template <typename T, int VEC>
static cudaError_t launch_stream_conv(const StreamConvParams& p, dim3 grid, cudaStream_t stream) {
  switch (p.n_taps) {
    case 2: return launch_pdl(stream_conv_kernel<T, VEC, 2>, grid, dim3(256), 0, stream, p);
    case 3: return launch_pdl(stream_conv_kernel<T, VEC, 3>, grid, dim3(256), 0, stream, p);
    case 4: return launch_pdl(stream_conv_kernel<T, VEC, 4>, grid, dim3(256), 0, stream, p);
    default: return launch_pdl(stream_conv_kernel<T, VEC, 0>, grid, dim3(256), 0, stream, p);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) embedding_stream_kernel(const int* __restrict__ ids, const T* __restrict__ table,
                                                                float* __restrict__ x, T* __restrict__ act, const int* __restrict__ positions,
                                                                const float* __restrict__ inv_freq, int W, int rows, float scale) {
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int id = ids[blockIdx.x];
  const bool ok = id >= 0 && id < rows;
  const T* src = table + static_cast<size_t>(ok ? id : 0) * W;
  const size_t base = static_cast<size_t>(blockIdx.x) * W;
  auto put = [&](int c, float add) {
    const float v = (ok ? to_f32(src[c]) * scale : 0.f) + add;
    x[base + c] = v;
    if (act != nullptr) act[base + c] = from_f32<T>(v);
  };
  if (inv_freq != nullptr) {
    const float pos = static_cast<float>(positions[blockIdx.x]);
    for (int i = blockIdx.y * 256 + threadIdx.x; 2 * i < W; i += 256 * gridDim.y) {
      float sn, cs;
      sincosf(pos * inv_freq[i], &sn, &cs);
      if (W % 2 == 0 && act == nullptr) {
        const float u = ok ? to_f32(src[2 * i]) * scale : 0.f, v = ok ? to_f32(src[2 * i + 1]) * scale : 0.f;
        *reinterpret_cast<float2*>(x + base + 2 * i) = make_float2(u + sn, v + cs);
        continue;
      }
      put(2 * i, sn);
      if (2 * i + 1 < W) put(2 * i + 1, cs);
    }
    return;
  }
  for (int c = threadIdx.x; c < W; c += 256) put(c, 0.f);
}

struct QkvPrepParams {
  const void* qkv;
  void* q_out;      // [M, n_q, dk]
  void* k_cache;    // [pages, n_kv, 16, dk]
  void* v_cache;    // [pages, n_kv, 16, dv]
  const int* positions;
  const long long* slots;     // page * 16 + offset, < 0 = do not store
  const float* inv_freq;      // [rot / 2]
  const float* q_norm_w;      // [n_q dk] or null
  const float* k_norm_w;      // [n_kv dk] or null
  int ld, n_q, n_kv, dk, dv, rot;
  int value_norm, append;
  float eps;
};

constexpr int kMaxRotPairs = 256;

// One CTA per token.
template <typename T>
__global__ void __launch_bounds__(256) qkv_prepare_kernel(QkvPrepParams p) {
  __shared__ float red[8];
  __shared__ float cs[kMaxRotPairs], sn[kMaxRotPairs];
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x;
  const int half = p.rot >> 1;
  const T* row = static_cast<const T*>(p.qkv) + static_cast<size_t>(m) * p.ld;
  const int qn = p.n_q * p.dk, kn = p.n_kv * p.dk;
  const long long slot = p.slots[m];
  const bool store = p.append && slot >= 0;
  const float pos = static_cast<float>(p.positions[m]);
  for (int i = threadIdx.x; i < half; i += 256) sincosf(pos * p.inv_freq[i], &sn[i], &cs[i]);
  float sq = 0.f, sk = 0.f;
  if (p.q_norm_w != nullptr)
    for (int c = threadIdx.x; c < qn; c += 256) {
      const float v = to_f32(row[c]);
      sq += v * v;
    }
  if (store && p.k_norm_w != nullptr)
    for (int c = threadIdx.x; c < kn; c += 256) {
      const float v = to_f32(row[qn + c]);
      sk += v * v;
    }
  const float q_inv = p.q_norm_w != nullptr ? 1.f / sqrtf(block_sum_f32(sq, red) / static_cast<float>(qn) + p.eps) : 1.f;
  const float k_inv = p.k_norm_w != nullptr && p.append ? 1.f / sqrtf(block_sum_f32(sk, red) / static_cast<float>(kn) + p.eps) : 1.f;
  __syncthreads();  // cs / sn
  const int per = p.dk - half;  // rotation pairs and pass-through elements of a head
  auto head = [&](const T* src, const float* w, float inv, int h, int j, T* dst) {
    const int c = h * p.dk + j;
    float u = to_f32(src[c]) * inv * (w != nullptr ? w[c] : 1.f);
    if (j < half) {
      const float v = to_f32(src[c + half]) * inv * (w != nullptr ? w[c + half] : 1.f);
      dst[j] = from_f32<T>(u * cs[j] - v * sn[j]);
      dst[j + half] = from_f32<T>(v * cs[j] + u * sn[j]);
    } else {
      dst[j + half] = from_f32<T>(to_f32(src[c + half]) * inv * (w != nullptr ? w[c + half] : 1.f));
    }
  };
  T* q = static_cast<T*>(p.q_out) + static_cast<size_t>(m) * qn;
  for (int i = threadIdx.x; i < p.n_q * per; i += 256) {
    const int h = i / per, j = i - h * per;
    head(row, p.q_norm_w, q_inv, h, j, q + static_cast<size_t>(h) * p.dk);
  }
  if (!store) return;
  const size_t page = static_cast<size_t>(slot >> 4);
  const int off = static_cast<int>(slot & 15);
  T* kc = static_cast<T*>(p.k_cache);
  for (int i = threadIdx.x; i < p.n_kv * per; i += 256) {
    const int h = i / per, j = i - h * per;
    head(row + qn, p.k_norm_w, k_inv, h, j, kc + ((page * p.n_kv + h) * 16 + off) * p.dk);
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  T* vc = static_cast<T*>(p.v_cache);
  for (int h = warp; h < p.n_kv; h += 8) {
    const T* src = row + qn + kn + static_cast<size_t>(h) * p.dv;
    T* dst = vc + ((page * p.n_kv + h) * 16 + off) * p.dv;
    float inv = 1.f;
    if (p.value_norm) {
      float ss = 0.f;
      for (int c = lane; c < p.dv; c += 32) {
        const float v = to_f32(src[c]);
        ss += v * v;
      }
      inv = 1.f / sqrtf(warp_sum_f32(ss) / static_cast<float>(p.dv) + p.eps);
    }
    for (int c = lane; c < p.dv; c += 32) dst[c] = from_f32<T>(to_f32(src[c]) * inv);
  }
}

}  // namespace eredu

using namespace eredu;

// y [M, W] bf16 (y_fp32 = 0) or fp32; w fp32 [1] (w_vec = 0) or [W]; residual, x_out fp32 [M, W] or null; act bf16 [M, W] or null.
extern "C" int eredu_rms_residual(const void* y, const float* w, const float* residual, float* x_out, void* act, int M, int W,
                                  int y_fp32, int w_vec, float eps, cudaStream_t stream) {
  if (M <= 0 || W <= 0) return 0;
  __nv_bfloat16* a = static_cast<__nv_bfloat16*>(act);
  const cudaError_t e = y_fp32 ? launch_rms_residual(static_cast<const float*>(y), w, w_vec, residual, x_out, a, M, W, eps, stream)
                               : launch_rms_residual(static_cast<const __nv_bfloat16*>(y), w, w_vec, residual, x_out, a, M, W, eps, stream);
  eredu_count_launches(1);
  return static_cast<int>(e);
}

// x, x_out, weight, bias fp32; y, rows, act bf16 (fp32 = 0) or fp32; k <= 32 routes per row; quads: rows are whole 16-byte pieces.
extern "C" int eredu_residual_norm(const float* x, const void* y, const void* rows, const int* route_pos, const float* route_w,
                                   const float* weight, const float* bias, float* x_out, void* act, int M, int W, int k, int fp32, int center,
                                   int quads, float eps, cudaStream_t stream) {
  if (M <= 0 || W <= 0) return 0;
  if (k < 0 || k > kMaxRoutes || (k > 0 && (rows == nullptr || route_pos == nullptr || route_w == nullptr)) ||
      (weight != nullptr && act == nullptr) || (x_out == nullptr && (y != nullptr || k > 0)))
    return -1;
  const ResidualNormParams p = {x, y, rows, route_pos, route_w, weight, bias, x_out, act, W, k, center, eps};
  const cudaError_t e = fp32 ? launch_residual_norm<float>(p, M, quads != 0, stream) : launch_residual_norm<__nv_bfloat16>(p, M, quads != 0, stream);
  eredu_count_launches(1);
  return static_cast<int>(e);
}

// x, x_out, weights fp32; y0, y1 (or null), act bf16 (fp32 = 0) or fp32; w0, w1: norms of the branches, both or neither null.
extern "C" int eredu_branch_norm(const float* x, const void* y0, const void* y1, const float* w0, const float* w1, const float* weight,
                                 const float* next, float* x_out, void* act, int M, int W, int fp32, int quads, float gain, float eps,
                                 cudaStream_t stream) {
  if (M <= 0 || W <= 0) return 0;
  if ((next != nullptr && act == nullptr) || (y1 != nullptr && (w0 == nullptr) != (w1 == nullptr))) return -1;
  const BranchNormParams p = {x, y0, y1, w0, w1, weight, next, x_out, act, W, gain, eps};
  const cudaError_t e = fp32 ? launch_branch_norm<float>(p, M, quads != 0, stream) : launch_branch_norm<__nv_bfloat16>(p, M, quads != 0, stream);
  eredu_count_launches(1);
  return static_cast<int>(e);
}

// weight, residual, x_out, taps, state fp32; y (or null), rows, act (or null) bf16 (fp32 = 0) or fp32; k <= 32 routes per row. taps: row m is
// the only row of sequence m; state may be null for one tap.
extern "C" int eredu_rms_routed_residual(const void* y, const void* rows, const int* route_pos, const float* route_w, const float* weight,
                                         const float* residual, float* x_out, void* act, const float* taps, float* state,
                                         const int* block_table, const int* page_to_slot, const long long* slots, int M, int W, int k,
                                         int n_taps, int state_elems, int max_pages, int fp32, int quads, float eps, cudaStream_t stream) {
  if (M <= 0 || W <= 0) return 0;
  if (k < 0 || k > kMaxRoutes || (k > 0 && (rows == nullptr || route_pos == nullptr || route_w == nullptr)) || (y == nullptr && k == 0) ||
      (taps != nullptr && (n_taps < 1 || act == nullptr || (n_taps > 1 && state == nullptr))) ||
      (state != nullptr && state_elems < (n_taps - 1) * W))
    return -1;
  const RaggedBatch seqs = {block_table, page_to_slot, nullptr, slots, M, 1, max_pages};
  const RoutedResidualParams p = {y, rows, route_pos, route_w, weight, residual, x_out, act, taps, state, seqs, n_taps, state_elems, W, k, eps};
  const bool q4 = quads != 0 && state_elems % 4 == 0;
  const cudaError_t e = fp32 ? launch_rms_routed_residual<float>(p, M, q4, stream) : launch_rms_routed_residual<__nv_bfloat16>(p, M, q4, stream);
  eredu_count_launches(1);
  return static_cast<int>(e);
}

// x fp32 [M, W]; act bf16 (fp32 = 0) or fp32; state may be null for one tap. max_rows: the most rows of a sequence.
extern "C" int eredu_stream_conv(const float* x, void* act, const float* taps, float* state, const int* block_table, const int* page_to_slot,
                                 const int* cu_q, const long long* slots, int batch, int q_per_seq, int max_rows, int max_pages, int W,
                                 int n_taps, int state_elems, int fp32, cudaStream_t stream) {
  if (batch <= 0 || max_rows <= 0 || W <= 0) return 0;
  if (n_taps < 1 || (n_taps > 1 && (state == nullptr || state_elems < (n_taps - 1) * W)) || batch > 65535) return -1;
  int tile = 16;
  while (tile < n_taps - 1 || (max_rows + tile - 1) / tile > 65535) tile *= 2;
  const RaggedBatch seqs = {block_table, page_to_slot, cu_q, slots, batch, q_per_seq, max_pages};
  const StreamConvParams p = {x, act, taps, state, seqs, W, n_taps, state_elems, tile};
  const int vec = W % 4 == 0 && state_elems % 4 == 0 ? 4 : 1;
  const dim3 grid((W + 256 * vec - 1) / (256 * vec), (max_rows + tile - 1) / tile, batch);
  cudaError_t e;
  if (vec == 4) e = fp32 ? launch_stream_conv<float, 4>(p, grid, stream) : launch_stream_conv<__nv_bfloat16, 4>(p, grid, stream);
  else e = fp32 ? launch_stream_conv<float, 1>(p, grid, stream) : launch_stream_conv<__nv_bfloat16, 1>(p, grid, stream);
  eredu_count_launches(1);
  return static_cast<int>(e);
}

// table [rows, W] bf16 or fp32, times scale; x fp32 [M, W]; act [M, W] in the table's dtype or null.
// inv_freq [(W + 1) / 2] or null: columns 2 i and 2 i + 1 get sin and cos of positions[m] * inv_freq[i] added.
extern "C" int eredu_embedding_stream(const int* ids, const void* table, float* x, void* act, const int* positions, const float* inv_freq,
                                      int M, int W, int rows, int fp32, float scale, cudaStream_t stream) {
  if (M <= 0 || W <= 0) return 0;
  cudaError_t e;
  // few rows: a sine and a cosine per thread
  const dim3 grid(M, inv_freq != nullptr && M <= 512 ? ((W + 1) / 2 + 255) / 256 : 1);
  if (fp32) e = launch_pdl(embedding_stream_kernel<float>, grid, dim3(256), 0, stream, ids, static_cast<const float*>(table), x,
                           static_cast<float*>(act), positions, inv_freq, W, rows, scale);
  else e = launch_pdl(embedding_stream_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, ids,
                      static_cast<const __nv_bfloat16*>(table), x, static_cast<__nv_bfloat16*>(act), positions, inv_freq, W, rows, scale);
  eredu_count_launches(1);
  return static_cast<int>(e);
}

extern "C" int eredu_qkv_prepare(const void* qkv, void* q_out, void* k_cache, void* v_cache, const int* positions,
                                 const long long* slots, const float* inv_freq, const float* q_norm_w, const float* k_norm_w, int M,
                                 int ld, int n_q, int n_kv, int dk, int dv, int rot, int value_norm, int append, int fp32, float eps,
                                 cudaStream_t stream) {
  if (M <= 0) return 0;
  if (rot < 0 || rot > dk || rot % 2 != 0 || rot / 2 > kMaxRotPairs) return -1;
  QkvPrepParams p;
  p.qkv = qkv;
  p.q_out = q_out;
  p.k_cache = k_cache;
  p.v_cache = v_cache;
  p.positions = positions;
  p.slots = slots;
  p.inv_freq = inv_freq;
  p.q_norm_w = q_norm_w;
  p.k_norm_w = k_norm_w;
  p.ld = ld;
  p.n_q = n_q;
  p.n_kv = n_kv;
  p.dk = dk;
  p.dv = dv;
  p.rot = rot;
  p.value_norm = value_norm;
  p.append = append;
  p.eps = eps;
  const cudaError_t e = fp32 ? launch_pdl(qkv_prepare_kernel<float>, dim3(M), dim3(256), 0, stream, p)
                             : launch_pdl(qkv_prepare_kernel<__nv_bfloat16>, dim3(M), dim3(256), 0, stream, p);
  eredu_count_launches(1);
  return static_cast<int>(e);
}
