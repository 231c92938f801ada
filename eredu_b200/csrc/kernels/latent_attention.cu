// Absorbed latent attention: every head of a token attends over the same cached rows [latent (rank) | key part (rot)]; scores use the
// whole row, the weighted sum the latent part. Queries q [rows, heads, rank + rot] are in latent space already; the result [rows,
// heads, rank] is expanded to values by the caller. Sliding window and sinks; decode steps and portions of prompts.
//
// The (token, head) pairs of a sequence are the rows of the tiles, token-major, so a CTA reads a cached row once for up to 64 heads.
// Eight warps = RG groups of 16 rows x CG groups of output columns. A step takes KT keys:
//   scores  : warp (rg, cg) forms 16 rows x KT / CG keys over the whole row width, left in shared memory as fp32
//   softmax : all threads, 256 / rows of them per row: running maximum and sum in registers, weights as bf16 and the rescale
//             factor of the row in shared memory
//   output  : warp (rg, cg) adds weights x latents for its rows and columns; the accumulator lives in registers
// Cached rows come page by page through a cp.async ring. Several splits of the keys form a thread-block cluster and combine
// their partial results through distributed shared memory.
#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/launch_count.h"
#include "../common/mma.cuh"
#include "../common/ptx.cuh"

namespace eredu {

using bf16 = __nv_bfloat16;

struct LatentAttnParams {
  const bf16* q;           // [total, H, D], D = rank + rot
  const bf16* cache;       // [pages * 16, D]
  bf16* out;               // [total, H, rank]
  const int* block_table;  // [B, max_pages]
  const int* seq_lens;     // [B] cached tokens including the new ones
  const int* cu_q;         // [B + 1] row offsets of the queries, or null: q_per_seq each
  const float* sinks;      // [H] or null
  int q_per_seq, max_pages, H, rank, D, splits, window;
  float scale_log2;
};

template <int RG>
struct LatentTile {
  static constexpr int kRows = RG * 16;
  static constexpr int kCg = 8 / RG;
  static constexpr int kKeys = RG == 1 ? 64 : 32;
  static constexpr int kStages = RG == 1 ? 2 : 3;
  static constexpr int kSw = kKeys / kCg;        // keys a warp scores: 8 or 16
  static constexpr int kTpr = 256 / kRows;       // softmax threads per row
  static constexpr int kKpt = kKeys / kTpr;      // keys each of them takes
};

__host__ __device__ inline int latent_width(int D) { return (D + 31) & ~31; }  // row width in shared memory, without the pad

template <int RG>
__host__ __device__ inline size_t latent_ring_bytes(int D) {
  using T = LatentTile<RG>;
  return static_cast<size_t>(T::kRows + T::kStages * T::kKeys) * (latent_width(D) + 8) * sizeof(bf16);
}
template <int RG>
__host__ __device__ inline size_t latent_smem_bytes(int D, int rank, int splits) {
  using T = LatentTile<RG>;
  const size_t ring = latent_ring_bytes<RG>(D), partial = splits > 1 ? static_cast<size_t>(T::kRows) * rank * sizeof(float) : 0;
  return (ring > partial ? ring : partial) + T::kRows * ((T::kKeys + 4) * sizeof(float) + (T::kKeys + 8) * sizeof(bf16) + 3 * sizeof(float));
}

__device__ __forceinline__ float ld_cluster_f32(uint32_t addr) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
  return v;
}
__device__ __forceinline__ float4 ld_cluster_f32x4(uint32_t addr) {
  float4 v;
  asm volatile("ld.shared::cluster.v4.f32 {%0, %1, %2, %3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(addr) : "memory");
  return v;
}

// NT: 8-column tiles of the output per warp (even). grid (splits, row tiles, B).
template <int RG, int NT>
__global__ void __launch_bounds__(256, 1) latent_attn_kernel(LatentAttnParams p) {
  using T = LatentTile<RG>;
  extern __shared__ __align__(16) uint8_t smem[];
  const int W = latent_width(p.D), S = W + 8;                       // row width and stride, elements
  bf16* q_s = reinterpret_cast<bf16*>(smem);                        // [rows][S]
  bf16* ring = q_s + T::kRows * S;                                  // [stages][keys][S]
  const size_t ring_bytes = latent_ring_bytes<RG>(p.D);
  const size_t part_bytes = p.splits > 1 ? static_cast<size_t>(T::kRows) * p.rank * sizeof(float) : 0;
  float* s_s = reinterpret_cast<float*>(smem + (ring_bytes > part_bytes ? ring_bytes : part_bytes));  // [rows][keys + 4]
  bf16* p_s = reinterpret_cast<bf16*>(s_s + T::kRows * (T::kKeys + 4));                                // [rows][keys + 8]
  float* corr_s = reinterpret_cast<float*>(p_s + T::kRows * (T::kKeys + 8));                           // [rows]
  float* m_s = corr_s + T::kRows;                                                                      // [rows]
  float* l_s = m_s + T::kRows;                                                                         // [rows]

  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.z, split = blockIdx.x;
  const int q0 = p.cu_q != nullptr ? p.cu_q[b] : b * p.q_per_seq;
  const int q_len = p.cu_q != nullptr ? p.cu_q[b + 1] - q0 : p.q_per_seq;
  const int row0 = blockIdx.y * T::kRows, rows = q_len * p.H;
  if (row0 >= rows) return;                                         // uniform over the cluster
  const int kv_len = p.seq_lens[b];
  const int pos0 = kv_len - q_len;
  const int last_row = min(rows, row0 + T::kRows) - 1;
  const int first_pos = pos0 + row0 / p.H, last_pos = pos0 + last_row / p.H;
  const int lo = p.window > 0 ? max(0, first_pos - p.window + 1) : 0, hi = last_pos + 1;
  const int per = ((hi - lo + p.splits - 1) / p.splits + T::kKeys - 1) / T::kKeys * T::kKeys;
  const int k_begin = lo + split * per, k_end = min(hi, k_begin + per);
  const int steps = k_end > k_begin ? (k_end - k_begin + T::kKeys - 1) / T::kKeys : 0;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rg = warp % RG, cg = warp / RG;
  const int g = lane >> 2, tig = lane & 3;
  const int* bt = p.block_table + static_cast<size_t>(b) * p.max_pages;
  const int chunks = W / 8, real = p.D / 8;

  for (int i = threadIdx.x; i < T::kRows * chunks; i += 256) {
    const int r = i / chunks, c = i - r * chunks;
    const bool ok = row0 + r < rows && c < real;
    const bf16* src = p.q + (static_cast<size_t>(q0) * p.H + row0 + (ok ? r : 0)) * p.D + (ok ? c * 8 : 0);
    cp_async16(q_s + r * S + c * 8, src, ok ? 16 : 0);
  }
  // a warp copies whole rows: the page lookup is one load per row
  auto load_keys = [&](int step) {
    bf16* dst = ring + (step % T::kStages) * T::kKeys * S;
#pragma unroll
    for (int i = 0; i < T::kKeys / 8; ++i) {
      const int r = warp + 8 * i, key = k_begin + step * T::kKeys + r;
      const bool in = key < k_end;
      const bf16* src = p.cache + (in ? (static_cast<size_t>(bt[key >> 4]) * 16 + (key & 15)) * p.D : 0);
      for (int c = lane; c < chunks; c += 32) {
        const bool ok = in && c < real;
        cp_async16(dst + r * S + c * 8, src + (ok ? c * 8 : 0), ok ? 16 : 0);
      }
    }
  };
#pragma unroll
  for (int s = 0; s < T::kStages - 1; ++s) {
    if (s < steps) load_keys(s);
    cp_async_commit();
  }
  // softmax role: row sr, keys [sk, sk + kKpt) of a step
  const int sr = threadIdx.x / T::kTpr, sk = (threadIdx.x % T::kTpr) * T::kKpt;
  const int s_pos = pos0 + min(row0 + sr, rows - 1) / p.H;
  const int s_low = p.window > 0 ? max(0, s_pos - p.window + 1) : 0;
  const bool s_live = row0 + sr < rows;
  float m = -INFINITY, l = 0.f;
  float o[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  const int tiles = p.rank / 8;
  const int tile0 = cg * NT;

  for (int step = 0; step < steps; ++step) {
    cp_async_wait<T::kStages - 2>();
    __syncthreads();                                                // keys landed; the stage read two barriers ago is free
    if (step + T::kStages - 1 < steps) load_keys(step + T::kStages - 1);
    cp_async_commit();
    const bf16* kt = ring + (step % T::kStages) * T::kKeys * S;
    float sc[2][4] = {};
    if constexpr (T::kSw == 16) {
#pragma unroll 4
      for (int ks = 0; ks < W / 16; ++ks) {
        uint32_t b0, b1, b2, b3, a0, a1, a2, a3;
        ldsm_x4(smem_u32(kt + (cg * 16 + (lane & 7) + (lane >> 4) * 8) * S + ks * 16 + ((lane >> 3) & 1) * 8), b0, b1, b2, b3);
        ldsm_x4(smem_u32(q_s + (rg * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * S + ks * 16 + (lane >> 4) * 8), a0, a1, a2, a3);
        mma16816(sc[0], a0, a1, a2, a3, b0, b1);
        mma16816(sc[1], a0, a1, a2, a3, b2, b3);
      }
    } else {
#pragma unroll 2
      for (int ks = 0; ks < W / 32; ++ks) {                         // 8 keys x two 16-wide pieces per load; two independent sums
        uint32_t b0, b1, b2, b3, a0, a1, a2, a3;
        ldsm_x4(smem_u32(kt + (cg * 8 + (lane & 7)) * S + ks * 32 + (lane >> 3) * 8), b0, b1, b2, b3);
        const bf16* qa = q_s + (rg * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * S + ks * 32 + (lane >> 4) * 8;
        ldsm_x4(smem_u32(qa), a0, a1, a2, a3);
        mma16816(sc[0], a0, a1, a2, a3, b0, b1);
        ldsm_x4(smem_u32(qa + 16), a0, a1, a2, a3);
        mma16816(sc[1], a0, a1, a2, a3, b2, b3);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) sc[0][e] += sc[1][e];
    }
#pragma unroll
    for (int j = 0; j < T::kSw / 8; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r)
        *reinterpret_cast<float2*>(s_s + (rg * 16 + g + r * 8) * (T::kKeys + 4) + cg * T::kSw + j * 8 + tig * 2) =
            make_float2(sc[j][2 * r], sc[j][2 * r + 1]);
    __syncthreads();
    {
      const int key0 = k_begin + step * T::kKeys + sk;
      float v[T::kKpt], mx = m;
#pragma unroll
      for (int i = 0; i < T::kKpt; ++i) {
        const int key = key0 + i;
        v[i] = s_live && key < k_end && key <= s_pos && key >= s_low ? s_s[sr * (T::kKeys + 4) + sk + i] * p.scale_log2 : -INFINITY;
        mx = fmaxf(mx, v[i]);
      }
#pragma unroll
      for (int d = 1; d < T::kTpr; d <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
      const float base = mx == -INFINITY ? 0.f : mx;
      const float corr = exp2f(m - base);                           // m = -inf: 0
      m = mx;
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < T::kKpt; i += 2) {
        const float e0 = exp2f(v[i] - base), e1 = exp2f(v[i + 1] - base);
        sum += e0 + e1;
        *reinterpret_cast<uint32_t*>(p_s + sr * (T::kKeys + 8) + sk + i) = pack_bf16x2(e0, e1);
      }
      l = l * corr + sum;                                           // this thread's share of the row
      if (threadIdx.x % T::kTpr == 0) corr_s[sr] = corr;
    }
    __syncthreads();
    const float c0 = corr_s[rg * 16 + g], c1 = corr_s[rg * 16 + g + 8];
    if (__any_sync(0xffffffffu, c0 != 1.f || c1 != 1.f)) {
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        o[i][0] *= c0;
        o[i][1] *= c0;
        o[i][2] *= c1;
        o[i][3] *= c1;
      }
    }
#pragma unroll
    for (int kk = 0; kk < T::kKeys / 16; ++kk) {
      uint32_t a0, a1, a2, a3;
      ldsm_x4(smem_u32(p_s + (rg * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * (T::kKeys + 8) + kk * 16 + (lane >> 4) * 8), a0, a1, a2, a3);
      const bf16* vrow = kt + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * S + (lane >> 4) * 8;
#pragma unroll
      for (int i = 0; i < NT; i += 2) {
        if (tile0 + i >= tiles) break;                              // warp-uniform
        uint32_t b0, b1, b2, b3;
        // the second tile of the last pair may lie behind the latent: it is inside the row's shared memory and not stored
        ldsm_x4_t(smem_u32(vrow + (tile0 + i) * 8), b0, b1, b2, b3);
        mma16816(o[i], a0, a1, a2, a3, b0, b1);
        mma16816(o[i + 1], a0, a1, a2, a3, b2, b3);
      }
    }
  }
  cp_async_wait<0>();
  // row sums over the threads of a row
#pragma unroll
  for (int d = 1; d < T::kTpr; d <<= 1) l += __shfl_xor_sync(0xffffffffu, l, d);
  __syncthreads();                                                  // every warp is done with the ring
  if (threadIdx.x % T::kTpr == 0) {
    m_s[sr] = m;
    l_s[sr] = l;
  }
  const size_t out_row0 = static_cast<size_t>(q0) * p.H + row0;
  // weight of a row's accumulator once the sink is counted: e^(m - M) / (l e^(m - M) + e^(sink - M)), M the larger of both
  auto finish = [&](int r, float mr, float lr) {
    if (p.sinks == nullptr) return lr > 0.f ? 1.f / lr : 0.f;
    const float sink = p.sinks[(row0 + r) % p.H] * 1.4426950408889634f;
    const float M = fmaxf(mr, sink);
    const float e = exp2f(mr - M);
    return e / (lr * e + exp2f(sink - M));
  };
  if (p.splits == 1) {
    __syncthreads();
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int row = rg * 16 + g + r * 8;
      if (row0 + row >= rows) continue;
      const float inv = finish(row, m_s[row], l_s[row]);
      bf16* dst = p.out + (out_row0 + row) * p.rank;
#pragma unroll
      for (int i = 0; i < NT; ++i)
        if (tile0 + i < tiles)
          *reinterpret_cast<uint32_t*>(dst + (tile0 + i) * 8 + tig * 2) = pack_bf16x2(o[i][2 * r] * inv, o[i][2 * r + 1] * inv);
    }
    return;
  }
  float* part = reinterpret_cast<float*>(smem);                     // [rows][rank], over the ring
#pragma unroll
  for (int r = 0; r < 2; ++r)
#pragma unroll
    for (int i = 0; i < NT; ++i)
      if (tile0 + i < tiles)
        *reinterpret_cast<float2*>(part + static_cast<size_t>(rg * 16 + g + r * 8) * p.rank + (tile0 + i) * 8 + tig * 2) =
            make_float2(o[i][2 * r], o[i][2 * r + 1]);
  cluster_arrive_release();
  cluster_wait_acquire();
  const uint32_t a_p = smem_u32(part), a_m = smem_u32(m_s), a_l = smem_u32(l_s);
  const int quads = p.rank / 4;
  for (int row = split * 8 + warp; row < T::kRows; row += 8 * p.splits) {  // a warp takes a row
    if (row0 + row >= rows) break;
    float M = -INFINITY;
    for (int sp = 0; sp < p.splits; ++sp) M = fmaxf(M, ld_cluster_f32(mapa_shared(a_m + row * 4, sp)));
    float L = 0.f;
    for (int sp = 0; sp < p.splits; ++sp) {
      const float ms = ld_cluster_f32(mapa_shared(a_m + row * 4, sp));
      L += ms == -INFINITY ? 0.f : ld_cluster_f32(mapa_shared(a_l + row * 4, sp)) * exp2f(ms - M);
    }
    const float inv = finish(row, M, L);
    for (int c = lane; c < quads; c += 32) {
      float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int sp = 0; sp < p.splits; ++sp) {
        const float ms = ld_cluster_f32(mapa_shared(a_m + row * 4, sp));
        const float e = ms == -INFINITY ? 0.f : exp2f(ms - M);
        const float4 v = ld_cluster_f32x4(mapa_shared(a_p + (row * p.rank + c * 4) * 4, sp));
        acc.x = fmaf(v.x, e, acc.x);
        acc.y = fmaf(v.y, e, acc.y);
        acc.z = fmaf(v.z, e, acc.z);
        acc.w = fmaf(v.w, e, acc.w);
      }
      store4(p.out + (out_row0 + row) * p.rank + c * 4, make_float4(acc.x * inv, acc.y * inv, acc.z * inv, acc.w * inv));
    }
  }
  cluster_arrive_release();  // done reading the peers' shared memory
  cluster_wait_acquire();    // and nobody reads this CTA's any more
}

template <int RG, int NT>
static cudaError_t launch_latent(const LatentAttnParams& p, dim3 grid, cudaStream_t stream) {
  const size_t smem = latent_smem_bytes<RG>(p.D, p.rank, p.splits);
  if (smem > 227 * 1024) return cudaErrorInvalidValue;
  static size_t configured[64] = {};
  int dev = 0;
  cudaError_t e = cudaGetDevice(&dev);
  if (e != cudaSuccess) return e;
  if (dev < 0 || dev >= 64) return cudaErrorInvalidDevice;
  if (configured[dev] < smem) {
    e = cudaFuncSetAttribute(latent_attn_kernel<RG, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return e;
    configured[dev] = smem;
  }
  cudaLaunchConfig_t lc = {};
  lc.gridDim = grid;
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
  if (p.splits > 1) {
    attr[n].id = cudaLaunchAttributeClusterDimension;
    attr[n].val.clusterDim.x = grid.x;
    attr[n].val.clusterDim.y = 1;
    attr[n].val.clusterDim.z = 1;
    ++n;
  }
  lc.attrs = attr;
  lc.numAttrs = n;
  return cudaLaunchKernelEx(&lc, latent_attn_kernel<RG, NT>, p);
}

template <int RG>
static cudaError_t launch_latent_rank(const LatentAttnParams& p, dim3 grid, cudaStream_t stream) {
  constexpr int kFull = 64 / (8 / RG);                              // 8-column tiles of a warp at rank 512
  const int need = (p.rank / 8 + 8 / RG - 1) / (8 / RG);
  if (need <= kFull / 4) return launch_latent<RG, kFull / 4>(p, grid, stream);
  if (need <= kFull / 2) return launch_latent<RG, kFull / 2>(p, grid, stream);
  return launch_latent<RG, kFull>(p, grid, stream);
}

}  // namespace eredu

using namespace eredu;

// rank, rot multiples of 8, rank <= 512; tile: rows of a CTA, 16, 32 or 64; splits <= 8.
extern "C" int eredu_latent_attn(const void* q, const void* cache, void* out, const int* block_table, const int* seq_lens, const int* cu_q,
                                 const float* sinks, int batch, int q_per_seq, int max_q, int max_pages, int heads, int rank, int rot,
                                 int tile, int splits, int window, float scale, cudaStream_t stream) {
  if (batch <= 0 || max_q <= 0) return 0;
  if (heads <= 0 || rank <= 0 || rank % 8 != 0 || rank > 512 || rot < 0 || rot % 8 != 0 || splits < 1 || splits > 8 || window < 0 || batch > 65535)
    return -1;
  LatentAttnParams p = {static_cast<const bf16*>(q), static_cast<const bf16*>(cache), static_cast<bf16*>(out), block_table, seq_lens, cu_q,
                        sinks, q_per_seq, max_pages, heads, rank, rank + rot, splits, window, scale * 1.4426950408889634f};
  const dim3 grid(splits, (max_q * heads + tile - 1) / tile, batch);
  if (grid.y > 65535) return -1;
  cudaError_t e;
  switch (tile) {
    case 16: e = launch_latent_rank<1>(p, grid, stream); break;
    case 32: e = launch_latent_rank<2>(p, grid, stream); break;
    case 64: e = launch_latent_rank<4>(p, grid, stream); break;
    default: return -1;
  }
  eredu_count_launches(1);
  return static_cast<int>(e);
}
