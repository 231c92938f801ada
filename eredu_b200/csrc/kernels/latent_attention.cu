// Absorbed latent attention: every head of a token attends over the same cached rows [latent (rank) | key part (rot)]; scores use the
// whole row, the weighted sum the latent part. Queries q [rows, heads, rank + rot] are in latent space already; the result [rows,
// heads, rank] is expanded to values by the caller. Sliding window and sinks; decode steps and portions of prompts.
//
// The (token, head) pairs of a sequence are the rows of the tiles, token-major, so a CTA reads a cached row once for up to 64 heads.
// Eight warps = RG groups of 16 rows x KG groups of keys x KH parts of the row width for the scores, RG x CG groups of output columns
// for the sum. A step takes 64 keys (32 with 64 rows):
//   scores  : a warp multiplies its rows, keys and part of the width; its queries stay in registers (RG < 4), so that only the keys are
//             read from shared memory. Partial sums go to shared memory as fp32
//   softmax : all threads, 256 / rows of them per row: running maximum and sum in registers, weights as bf16 and the rescale
//             factor of the row in shared memory
//   output  : warp (rg, cg) adds weights x latents for its rows and columns; the accumulator lives in registers
// Cached rows arrive by bulk copies, one per row (a page is 16 rows, but a window may start inside one), into a ring of
// slots of 32 rows. Several splits of the keys form a thread-block cluster and combine their partial results through distributed
// shared memory. Waits are bounded: on expiry the status word is set, the remaining waits are skipped, and the CTA leaves through the
// common exit after one more bounded wait for its copies.
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
  int* status;
};

constexpr int kSlot = 32;                        // cached rows of a ring slot

template <int RG>
struct LatentTile {
  static constexpr int kRows = RG * 16;
  static constexpr int kCg = 8 / RG;                    // column groups of the output
  static constexpr int kKh = RG < 4 ? 2 : 1;            // parts of the row width in the scores
  static constexpr int kKg = 8 / RG / kKh;              // groups of keys in the scores
  static constexpr int kKeys = RG < 4 ? 64 : 32;        // keys of a step
  static constexpr int kPer = kKeys / kSlot;            // slots of a step
  static constexpr int kSlots = RG < 4 ? 4 : 3;
  static constexpr int kKw = kKeys / kKg;               // keys a warp scores: 16 or 32
  static constexpr int kTpr = 256 / kRows;              // softmax threads per row
  static constexpr int kKpt = kKeys / kTpr;             // keys each of them takes
  static constexpr int kSStride = kKeys + 4, kPStride = kKeys + 8;
};

__host__ __device__ inline int latent_width(int D) { return (D + 31) & ~31; }  // row width in shared memory, without the pad

template <int RG>
__host__ __device__ inline size_t latent_ring_bytes(int D) {
  using T = LatentTile<RG>;
  return static_cast<size_t>(T::kRows + T::kSlots * kSlot) * (latent_width(D) + 8) * sizeof(bf16);
}
template <int RG>
__host__ __device__ inline size_t latent_smem_bytes(int D, int rank, int splits) {
  using T = LatentTile<RG>;
  const size_t ring = latent_ring_bytes<RG>(D), partial = splits > 1 ? static_cast<size_t>(T::kRows) * rank * sizeof(float) : 0;
  return (ring > partial ? ring : partial) + T::kRows * (T::kKh * T::kSStride * sizeof(float) + T::kPStride * sizeof(bf16) + 3 * sizeof(float));
}

// `bytes` (a multiple of 16) from 16-byte aligned global memory into this CTA's shared memory; counts on `bar` when it has landed.
__device__ __forceinline__ void bulk_load(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(dst)), "l"(src), "r"(bytes),
               "r"(smem_u32(bar))
               : "memory");
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

// TIER 1 / 2 / 4: latents of up to 128 / 256 / 512 entries in rows of up to 192 / 320 / 640. grid (splits, row tiles, B).
template <int RG, int TIER>
__global__ void __launch_bounds__(256, RG < 4 && TIER < 4 ? 2 : 1) latent_attn_kernel(LatentAttnParams p) {
  using T = LatentTile<RG>;
  constexpr int NT = 2 * TIER * RG;                                 // 8-column tiles of the output per warp
  constexpr bool kQReg = RG < 4;
  constexpr int kQs = kQReg ? (TIER == 1 ? 12 : TIER == 2 ? 20 : 40) / T::kKh : 1;  // 16-wide pieces of a warp's part
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ uint64_t full[T::kSlots];
  const int W = latent_width(p.D), S = W + 8;                       // row width and stride, elements
  bf16* q_s = reinterpret_cast<bf16*>(smem);                        // [rows][S]
  bf16* ring = q_s + T::kRows * S;                                  // [slots][kSlot][S]
  const size_t ring_bytes = latent_ring_bytes<RG>(p.D);
  const size_t part_bytes = p.splits > 1 ? static_cast<size_t>(T::kRows) * p.rank * sizeof(float) : 0;
  float* s_s = reinterpret_cast<float*>(smem + (ring_bytes > part_bytes ? ring_bytes : part_bytes));  // [parts][rows][kSStride]
  bf16* p_s = reinterpret_cast<bf16*>(s_s + T::kKh * T::kRows * T::kSStride);                          // [rows][kPStride]
  float* corr_s = reinterpret_cast<float*>(p_s + T::kRows * T::kPStride);                              // [rows]
  float* m_s = corr_s + T::kRows;                                                                      // [rows]
  float* l_s = m_s + T::kRows;                                                                         // [rows]

  pdl_launch_early();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int i = 0; i < T::kSlots; ++i) mbar_init(&full[i], 1);
    fence_mbar_init();
  }
  // the columns behind the row's own are zero in every slot; copies never touch them
  const int chunks = W / 8, real = p.D / 8;
  for (int i = threadIdx.x; i < T::kSlots * kSlot * (chunks - real); i += 256) {
    const int r = i / (chunks - real), c = real + i % (chunks - real);
    *reinterpret_cast<uint4*>(ring + r * S + c * 8) = make_uint4(0u, 0u, 0u, 0u);
  }
  __syncthreads();
  // Only the queries come from the kernel in front of this one: lengths, page tables and cached rows are older, so the rows start on their
  // way before the wait. (A kernel starts once all CTAs in front have passed their own wait, that is, once everything before those is
  // complete; not so when dependents are released early.)
  if (EREDU_PDL_EARLY) pdl_wait();
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
  const int rg = warp % RG, cg = warp / RG;
  const int kg = cg % T::kKg, kh = cg / T::kKg;                     // scores: group of keys, part of the width
  const int g = lane >> 2, tig = lane & 3;
  const int* bt = p.block_table + static_cast<size_t>(b) * p.max_pages;

  // ---- copies: the first lanes of every warp bring its share of a step's rows, one bulk copy each. Rows behind the last key repeat it
  // (they are masked).
  const uint32_t row_bytes = static_cast<uint32_t>(p.D) * sizeof(bf16);
  constexpr int kShare = T::kKeys / 8;                              // rows of a step a warp brings
  const int my_row = warp * kShare + lane;
  int page = 0;
  auto find_page = [&](int step) {                                  // one step ahead of the copies
    if (step < steps && lane < kShare) page = bt[min(k_begin + step * T::kKeys + my_row, k_end - 1) >> 4];
  };
  auto load_step = [&](int step) {
    if (step >= steps) return;
    const int slot0 = step * T::kPer % T::kSlots;
    if (threadIdx.x == 0) {
#pragma unroll
      for (int i = 0; i < T::kPer; ++i) mbar_arrive_expect_tx(&full[slot0 + i], kSlot * row_bytes);
    }
    if (lane < kShare) {
      const int key = min(k_begin + step * T::kKeys + my_row, k_end - 1);
      bulk_load(ring + (slot0 * kSlot + my_row) * S, p.cache + (static_cast<size_t>(page) * 16 + (key & 15)) * p.D, row_bytes,
                &full[slot0 + my_row / kSlot]);
    }
    find_page(step + 1);
  };
  constexpr int kAhead = T::kSlots / T::kPer;                       // steps in flight
  find_page(0);
#pragma unroll
  for (int s = 0; s < kAhead; ++s) load_step(s);
  pdl_wait();
  pdl_launch_dependents();
  for (int i = threadIdx.x; i < T::kRows * chunks; i += 256) {
    const int r = i / chunks, c = i - r * chunks;
    const bool ok = row0 + r < rows && c < real;
    const bf16* src = p.q + (static_cast<size_t>(q0) * p.H + row0 + (ok ? r : 0)) * p.D + (ok ? c * 8 : 0);
    cp_async16(q_s + r * S + c * 8, src, ok ? 16 : 0);
  }
  cp_async_commit();
  // softmax role: row sr, keys [sk, sk + kKpt) of a step
  const int sr = threadIdx.x / T::kTpr, sk = (threadIdx.x % T::kTpr) * T::kKpt;
  const int s_pos = pos0 + min(row0 + sr, rows - 1) / p.H;
  const int s_low = p.window > 0 ? max(0, s_pos - p.window + 1) : 0;
  // first and last step this row can see, relative to k_begin: keys outside [s_first, s_last] are masked
  const int s_first = row0 + sr < rows ? s_low - k_begin : 0x3fffffff, s_last = min(s_pos, k_end - 1) - k_begin;
  float m = -INFINITY, l = 0.f;
  float o[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  const int tiles = p.rank / 8;
  const int tile0 = cg * NT;
  const int parts = W / 16 / T::kKh;                                // 16-wide pieces of a warp's part of the width
  const int w0 = kh * parts * 16;
  const bf16* q_row = q_s + (rg * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * S + w0 + (lane >> 4) * 8;
  uint32_t qf[kQs][4];
  cp_async_wait<0>();
  __syncthreads();
  if (kQReg) {
#pragma unroll
    for (int i = 0; i < kQs; ++i)
      if (i < parts) ldsm_x4(smem_u32(q_row + i * 16), qf[i][0], qf[i][1], qf[i][2], qf[i][3]);
      else qf[i][0] = qf[i][1] = qf[i][2] = qf[i][3] = 0u;          // behind the row: the product with whatever is read adds nothing
  }

  bool live = true;
  for (int step = 0; step < steps; ++step) {
    const int slot0 = step * T::kPer % T::kSlots;
    const uint32_t parity = (step * T::kPer / T::kSlots) & 1;
#pragma unroll
    for (int i = 0; i < T::kPer; ++i) live = live && mbar_wait(&full[slot0 + i], parity, p.status, kStatusTmaFullTimeout);
    const bf16* kt = ring + slot0 * kSlot * S;
    constexpr int KT8 = T::kKw / 8;                                 // 8-key tiles of a warp
    float sc[2][KT8][4] = {};                                       // even and odd pieces apart
    const bf16* k_row = kt + (kg * T::kKw + (lane & 7) + (lane >> 4) * 8) * S + w0 + ((lane >> 3) & 1) * 8;
    // fragments are loaded in groups ahead of their products: with two warps per scheduler nothing else hides the latency
    if constexpr (kQReg) {
      constexpr int G = T::kKw == 16 ? 5 : 2;
#pragma unroll
      for (int i0 = 0; i0 < kQs; i0 += G) {
        uint32_t kf[G][KT8 / 2][4];
#pragma unroll
        for (int i = 0; i < G; ++i)
#pragma unroll
          for (int t = 0; t < KT8 / 2; ++t)
            if (i0 + i < kQs)
              ldsm_x4(smem_u32(k_row + t * 16 * S + min(i0 + i, parts - 1) * 16), kf[i][t][0], kf[i][t][1], kf[i][t][2], kf[i][t][3]);
#pragma unroll
        for (int i = 0; i < G; ++i)
#pragma unroll
          for (int t = 0; t < KT8 / 2; ++t)
            if (i0 + i < kQs) {
              const uint32_t* q = qf[i0 + i];
              mma16816(sc[(i0 + i) & 1][2 * t], q[0], q[1], q[2], q[3], kf[i][t][0], kf[i][t][1]);
              mma16816(sc[(i0 + i) & 1][2 * t + 1], q[0], q[1], q[2], q[3], kf[i][t][2], kf[i][t][3]);
            }
      }
    } else {
#pragma unroll 2
      for (int i0 = 0; i0 < parts; i0 += 2) {                       // W is a multiple of 32: an even number of pieces
        uint32_t kf[2][4], a[2][4];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          ldsm_x4(smem_u32(k_row + (i0 + i) * 16), kf[i][0], kf[i][1], kf[i][2], kf[i][3]);
          ldsm_x4(smem_u32(q_row + (i0 + i) * 16), a[i][0], a[i][1], a[i][2], a[i][3]);
        }
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          mma16816(sc[i][0], a[i][0], a[i][1], a[i][2], a[i][3], kf[i][0], kf[i][1]);
          mma16816(sc[i][1], a[i][0], a[i][1], a[i][2], a[i][3], kf[i][2], kf[i][3]);
        }
      }
    }
#pragma unroll
    for (int t = 0; t < KT8; ++t)
#pragma unroll
      for (int r = 0; r < 2; ++r)
        *reinterpret_cast<float2*>(s_s + (kh * T::kRows + rg * 16 + g + r * 8) * T::kSStride + kg * T::kKw + t * 8 + tig * 2) =
            make_float2(sc[0][t][2 * r] + sc[1][t][2 * r], sc[0][t][2 * r + 1] + sc[1][t][2 * r + 1]);
    __syncthreads();
    {
      const int key0 = step * T::kKeys + sk;
      const float* row = s_s + sr * T::kSStride + sk;
      float v[T::kKpt], mx = m;
#pragma unroll
      for (int i = 0; i < T::kKpt; ++i) {
        float sum = row[i];
        if (T::kKh == 2) sum += row[T::kRows * T::kSStride + i];
        v[i] = key0 + i >= s_first && key0 + i <= s_last ? sum * p.scale_log2 : -INFINITY;
        mx = fmaxf(mx, v[i]);
      }
#pragma unroll
      for (int d = 1; d < T::kTpr; d <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
      const float base = mx == -INFINITY ? 0.f : mx;
      const float corr = ex2_approx(m - base);                      // m = -inf: 0
      m = mx;
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < T::kKpt; i += 2) {
        const float e0 = ex2_approx(v[i] - base), e1 = ex2_approx(v[i + 1] - base);
        sum += e0 + e1;
        *reinterpret_cast<uint32_t*>(p_s + sr * T::kPStride + sk + i) = pack_bf16x2(e0, e1);
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
    {
      // tile pairs behind the latent repeat the last one (and are not stored); the second tile of the last pair may lie behind it, inside
      // the row's shared memory
      constexpr int G = NT / 2 < 4 ? NT / 2 : 4;
      const bf16* v0 = kt + ((lane & 7) + ((lane >> 3) & 1) * 8) * S + (lane >> 4) * 8;
      uint32_t pf[T::kKeys / 16][4];
#pragma unroll
      for (int kk = 0; kk < T::kKeys / 16; ++kk)
        ldsm_x4(smem_u32(p_s + (rg * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * T::kPStride + kk * 16 + (lane >> 4) * 8), pf[kk][0], pf[kk][1],
                pf[kk][2], pf[kk][3]);
#pragma unroll
      for (int kk = 0; kk < T::kKeys / 16; ++kk)
#pragma unroll
        for (int i0 = 0; i0 < NT / 2; i0 += G) {
          uint32_t vf[G][4];
#pragma unroll
          for (int i = 0; i < G; ++i)
            ldsm_x4_t(smem_u32(v0 + kk * 16 * S + min(tile0 + 2 * (i0 + i), (tiles - 1) & ~1) * 8), vf[i][0], vf[i][1], vf[i][2], vf[i][3]);
#pragma unroll
          for (int i = 0; i < G; ++i) {
            mma16816(o[2 * (i0 + i)], pf[kk][0], pf[kk][1], pf[kk][2], pf[kk][3], vf[i][0], vf[i][1]);
            mma16816(o[2 * (i0 + i) + 1], pf[kk][0], pf[kk][1], pf[kk][2], pf[kk][3], vf[i][2], vf[i][3]);
          }
        }
    }
    __syncthreads();                                                // the step's slots, scores and weights are free
    load_step(step + kAhead);
  }
  if (!live)                                                        // a copy is late: leave it time to land before the CTA goes
    for (int i = 0; i < T::kSlots; ++i) mbar_wait(&full[i], ((steps * T::kPer - 1 - i) / T::kSlots) & 1, p.status, kStatusTmaFullTimeout);
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
  // weight of every split's partial row, by one thread per row; then all threads of the cluster share the rows' columns
  constexpr int kMaxSplits = 8;
  float* wgt = s_s;                                                 // [rows][kMaxSplits]
  if (static_cast<int>(threadIdx.x) < T::kRows && row0 + static_cast<int>(threadIdx.x) < rows) {
    const int row = threadIdx.x;
    float ms[kMaxSplits], ls[kMaxSplits], M = -INFINITY, L = 0.f;
#pragma unroll
    for (int sp = 0; sp < kMaxSplits; ++sp) {
      const uint32_t from = sp < p.splits ? sp : 0;
      ms[sp] = ld_cluster_f32(mapa_shared(a_m + row * 4, from));
      ls[sp] = ld_cluster_f32(mapa_shared(a_l + row * 4, from));
    }
#pragma unroll
    for (int sp = 0; sp < kMaxSplits; ++sp)
      if (sp < p.splits) M = fmaxf(M, ms[sp]);
#pragma unroll
    for (int sp = 0; sp < kMaxSplits; ++sp) {
      ms[sp] = sp < p.splits && ms[sp] != -INFINITY ? ex2_approx(ms[sp] - M) : 0.f;
      L += ms[sp] * ls[sp];
    }
    const float inv = finish(row, M, L);
#pragma unroll
    for (int sp = 0; sp < kMaxSplits; ++sp) wgt[row * kMaxSplits + sp] = ms[sp] * inv;
  }
  __syncthreads();
  const int quads = p.rank / 4, total = min(T::kRows, rows - row0) * quads;
  for (int i = split * 256 + threadIdx.x; i < total; i += 256 * p.splits) {
    const int row = i / quads, c = i - row * quads;
    float4 v[kMaxSplits];
#pragma unroll
    for (int sp = 0; sp < kMaxSplits; ++sp)
      if (sp < p.splits) v[sp] = ld_cluster_f32x4(mapa_shared(a_p + (row * p.rank + c * 4) * 4, sp));
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int sp = 0; sp < kMaxSplits; ++sp) {
      if (sp >= p.splits) break;
      const float e = wgt[row * kMaxSplits + sp];
      acc = make_float4(fmaf(v[sp].x, e, acc.x), fmaf(v[sp].y, e, acc.y), fmaf(v[sp].z, e, acc.z), fmaf(v[sp].w, e, acc.w));
    }
    store4(p.out + (out_row0 + row) * p.rank + c * 4, acc);
  }
  cluster_arrive_release();  // done reading the peers' shared memory
  cluster_wait_acquire();    // and nobody reads this CTA's any more
}

template <int RG, int TIER>
static cudaError_t launch_latent(const LatentAttnParams& p, dim3 grid, cudaStream_t stream) {
  const size_t smem = latent_smem_bytes<RG>(p.D, p.rank, p.splits);
  if (smem > 227 * 1024) return cudaErrorInvalidValue;
  static size_t configured[64] = {};
  int dev = 0;
  cudaError_t e = cudaGetDevice(&dev);
  if (e != cudaSuccess) return e;
  if (dev < 0 || dev >= 64) return cudaErrorInvalidDevice;
  if (configured[dev] < smem) {
    e = cudaFuncSetAttribute(latent_attn_kernel<RG, TIER>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
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
  return cudaLaunchKernelEx(&lc, latent_attn_kernel<RG, TIER>, p);
}

template <int RG>
static cudaError_t launch_latent_rank(const LatentAttnParams& p, dim3 grid, cudaStream_t stream) {
  const int W = latent_width(p.D);
  if (p.rank <= 128 && W <= 192) return launch_latent<RG, 1>(p, grid, stream);
  if (p.rank <= 256 && W <= 320) return launch_latent<RG, 2>(p, grid, stream);
  return launch_latent<RG, 4>(p, grid, stream);
}

}  // namespace eredu

using namespace eredu;

// rank, rot multiples of 8, rank <= 512, rank + rot <= 640; tile: rows of a CTA, 16, 32 or 64; splits <= 8.
extern "C" int eredu_latent_attn(const void* q, const void* cache, void* out, const int* block_table, const int* seq_lens, const int* cu_q,
                                 const float* sinks, int batch, int q_per_seq, int max_q, int max_pages, int heads, int rank, int rot,
                                 int tile, int splits, int window, float scale, int* status, cudaStream_t stream) {
  if (batch <= 0 || max_q <= 0) return 0;
  if (heads <= 0 || rank <= 0 || rank % 8 != 0 || rank > 512 || rot < 0 || rot % 8 != 0 || rank + rot > 640 || splits < 1 || splits > 8 || window < 0 || batch > 65535)
    return -1;
  LatentAttnParams p = {static_cast<const bf16*>(q), static_cast<const bf16*>(cache), static_cast<bf16*>(out), block_table, seq_lens, cu_q,
                        sinks, q_per_seq, max_pages, heads, rank, rank + rot, splits, window, scale * 1.4426950408889634f, status};
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
