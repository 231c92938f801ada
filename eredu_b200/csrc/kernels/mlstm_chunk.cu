// mLSTM over long portions, chunk-parallel on the tensor cores (recurrence and layout: mlstm.cu).
//
// Inside a chunk of 64 tokens let b_t be the log forget gates summed up to t, a_s = i_s - b_s, and M_t = max(m_in, max_{s <= t} a_s)
// with m_in the running maximum that enters the chunk. Then m_t = b_t + M_t and
//   S_t^T q = e^(m_in - M_t) S_in^T q + sum_{s <= t} e^(a_s - M_t) (q . k_s) v_s,   n_t . q the same with n_in and 1 for v_s
// so every exponent is <= 0. Three launches do all chunks of all sequences and heads at once; only a scan over the states is sequential:
//   1. mlstm_chunk_state: what a chunk adds, sum_s e^(b_end + a_s - m_loc) k_s v_s^T (and without v), with its own scale m_loc
//   2. mlstm_chunk_scan:  per element the state that enters every chunk, over the contributions in place
//   3. mlstm_chunk_out:   outputs, normaliser, per-head norm and gate
// The products run on bf16 tensor cores without giving up 32-bit accuracy: every fp32 factor (gated keys, gated scores, the state) is
// split into two bf16 terms, hi + lo, and both products are added; queries, keys and values are bf16 to begin with. The scan stores
// four entries of the entering state as [hi x 4 | lo x 4] in the place of their fp32 values, so the output kernel multiplies both
// terms in one pass over twice as many columns and adds neighbouring results.
// Logarithms are to base 2 here, natural in the state.
#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/launch_count.h"
#include "../common/mma.cuh"
#include "../common/ptx.cuh"
#include "mlstm.h"

namespace eredu {

using bf16 = __nv_bfloat16;

constexpr int kC = 64, kThr = 256;
constexpr int kMaxKey = 256, kTileV = 128, kMaxTiles = 8;
constexpr int kPStride = kC + 8;
constexpr int kStageRows = 32;
constexpr float kLog2e = 1.4426950408889634f;

__host__ __device__ inline int key_pad(int dk) { return (dk + 15) & ~15; }

struct ChunkView {
  float* cells;      // [chunks][H (dk dv + dk)]: contributions, then entering states; per chunk memory [H, dk, dv], normaliser [H, dk]
  float2* scale;     // [chunks][H]: log forget gate of the chunk, log scale of its contribution
  float* m_in;       // [chunks][H]
};

// Unique over the batch; a sequence has one cell more than chunks.
__device__ __forceinline__ int chunk_cell(const RaggedSeq& s, int b, int c) { return s.row0 / kC + 2 * b + c; }

__device__ __forceinline__ float cluster_f32(uint32_t addr) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
  return v;
}

__device__ __forceinline__ void split_pair(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(a, b);
  lo = pack_bf16x2(a - bf16_lo(hi), b - bf16_hi(hi));
}

struct GateSmem {
  float b[kC], a[kC], top[kC];   // summed log forget gates, a_s, max over s <= t of a_s
};

// Gates of the chunk's tokens by the first two warps; tokens behind the portion neither forget nor add. Ends with a barrier.
__device__ __forceinline__ void chunk_gates(const MlstmParams<bf16>& p, GateSmem& gs, const RaggedSeq& seq, int h, int t0) {
  __shared__ float half_b, half_top;
  const int t = threadIdx.x, lane = t & 31;
  float b = 0.f, li = -INFINITY, top = 0.f;
  if (t < kC) {
    if (t0 + t < seq.rows) {
      const float2 g = mlstm_gates(p.gates + static_cast<size_t>(seq.row0 + t0 + t) * p.ldg, p.H, h, p.cap);
      li = g.x * kLog2e;
      b = g.y * kLog2e;
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, b, o);
      if (lane >= o) b += up;
    }
    if (t == 31) half_b = b;
  }
  __syncthreads();
  if (t < kC) {
    if (t >= 32) b += half_b;
    top = li - b;
    gs.b[t] = b;
    gs.a[t] = top;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, top, o);
      if (lane >= o) top = fmaxf(top, up);
    }
    if (t == 31) half_top = top;
  }
  __syncthreads();
  if (t < kC) gs.top[t] = t >= 32 ? fmaxf(top, half_top) : top;
  __syncthreads();
}

// `rows` of 16-byte pieces into shared memory, zero where the source ends.
__device__ __forceinline__ void copy_tile(bf16* dst, int stride, const bf16* src, long long ld, int rows, int live_rows, int pieces, int live_pieces) {
  for (int i = threadIdx.x; i < rows * pieces; i += kThr) {
    const int r = i / pieces, c = i - r * pieces;
    const bool ok = r < live_rows && c < live_pieces;
    cp_async16(dst + r * stride + c * 8, ok ? src + r * ld + c * 8 : src, ok ? 16 : 0);
  }
}

struct TileGeom {
  int h, b, c0, width;      // head, sequence, first value column and width of this CTA's tile
};
__device__ __forceinline__ TileGeom tile_geom(const MlstmParams<bf16>& p, int tile_w) {
  TileGeom g;
  g.h = blockIdx.z % p.H;
  g.b = blockIdx.z / p.H;
  g.c0 = blockIdx.x * tile_w;
  g.width = min(tile_w, p.dv - g.c0);
  return g;
}

// ---------------------------------------------------------------- 1. contributions of the chunks
// grid (value tiles, chunks, H * B). NT: 8-column tiles per warp.
template <int NT>
__global__ void __launch_bounds__(kThr, 2) mlstm_chunk_state_kernel(MlstmParams<bf16> p, ChunkView ws, int tile_w) {
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ GateSmem gs;
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const TileGeom tg = tile_geom(p, tile_w);
  const RaggedSeq seq = ragged_seq(p.seqs, tg.b);
  const int t0 = blockIdx.y * kC;
  if (!seq.live || t0 >= seq.rows) return;  // uniform
  const int dkp = key_pad(p.dk), ks = dkp + 8, vs = tile_w + 8;
  bf16* kh = reinterpret_cast<bf16*>(smem);          // [64][ks] keys, then the gated keys' hi terms
  bf16* kl = kh + kC * ks;                           // [64][ks] lo terms
  bf16* v = kl + kC * ks;                            // [64][vs]
  const int n = min(kC, seq.rows - t0);
  const int qk = p.H * p.dk;
  const bf16* rows = p.proj + static_cast<size_t>(seq.row0 + t0) * p.ld;
  copy_tile(kh, ks, rows + qk + tg.h * p.dk, p.ld, kC, n, dkp / 8, p.dk / 8);
  copy_tile(v, vs, rows + 2 * qk + tg.h * p.dv + tg.c0, p.ld, kC, n, tg.width / 8, tg.width / 8);
  cp_async_commit();
  chunk_gates(p, gs, seq, tg.h, t0);
  cp_async_wait<0>();
  __syncthreads();
  const float end = gs.b[kC - 1], m_loc = end + gs.top[kC - 1];
  const size_t chunk = chunk_cell(seq, tg.b, blockIdx.y);
  const size_t per_chunk = static_cast<size_t>(p.H) * p.dk * (p.dv + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int t = warp; t < kC; t += 8) {
    const float w = ex2_approx(end + gs.a[t] - m_loc);            // a = -inf behind the portion: 0
    for (int c = lane * 2; c < dkp; c += 64) {
      const uint32_t kk = *reinterpret_cast<const uint32_t*>(kh + t * ks + c);
      uint32_t hi, lo;
      split_pair(bf16_lo(kk) * w, bf16_hi(kk) * w, hi, lo);
      *reinterpret_cast<uint32_t*>(kh + t * ks + c) = hi;
      *reinterpret_cast<uint32_t*>(kl + t * ks + c) = lo;
    }
  }
  __syncthreads();
  if (blockIdx.x == 0) {
    if (threadIdx.x == 0) ws.scale[chunk * p.H + tg.h] = make_float2(end, m_loc);
    float* nd = ws.cells + chunk * per_chunk + static_cast<size_t>(p.H) * p.dk * p.dv + static_cast<size_t>(tg.h) * p.dk;
    for (int c = threadIdx.x; c < p.dk; c += kThr) {
      float sum = 0.f;
      for (int t = 0; t < kC; ++t) sum += to_f32(kh[t * ks + c]) + to_f32(kl[t * ks + c]);
      nd[c] = sum;
    }
  }
  const int g = lane >> 2, tig = lane & 3;
  const int nt = tg.width / 8;
  uint32_t vf[NT][8];
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    const int tile = min(warp + 8 * j, nt - 1);
#pragma unroll
    for (int half = 0; half < 2; ++half)
      ldsm_x4_t(smem_u32(v + (half * 32 + (lane & 7) + ((lane >> 3) & 1) * 8 + (lane >> 4) * 16) * vs + tile * 8), vf[j][4 * half],
                vf[j][4 * half + 1], vf[j][4 * half + 2], vf[j][4 * half + 3]);
  }
  float* out = ws.cells + chunk * per_chunk + static_cast<size_t>(tg.h) * p.dk * p.dv + tg.c0;
  for (int mt = 0; mt < dkp / 16; ++mt) {
    float acc[NT][4];
#pragma unroll
    for (int j = 0; j < NT; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      const int off = (kk * 16 + (lane & 7) + (lane >> 4) * 8) * ks + mt * 16 + ((lane >> 3) & 1) * 8;
      uint32_t a0, a1, a2, a3;
      ldsm_x4_t(smem_u32(kh + off), a0, a1, a2, a3);
#pragma unroll
      for (int j = 0; j < NT; ++j) mma16816(acc[j], a0, a1, a2, a3, vf[j][2 * kk], vf[j][2 * kk + 1]);
      ldsm_x4_t(smem_u32(kl + off), a0, a1, a2, a3);
#pragma unroll
      for (int j = 0; j < NT; ++j) mma16816(acc[j], a0, a1, a2, a3, vf[j][2 * kk], vf[j][2 * kk + 1]);
    }
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int tile = warp + 8 * j, r = mt * 16 + g;
      if (tile >= nt) continue;
      if (r < p.dk) *reinterpret_cast<float2*>(out + static_cast<size_t>(r) * p.dv + tile * 8 + tig * 2) = make_float2(acc[j][0], acc[j][1]);
      if (r + 8 < p.dk) *reinterpret_cast<float2*>(out + static_cast<size_t>(r + 8) * p.dv + tile * 8 + tig * 2) = make_float2(acc[j][2], acc[j][3]);
    }
  }
}

// ---------------------------------------------------------------- 2. the state that enters every chunk
// One thread per four elements of memory and normaliser of one sequence, which lie in a chunk's cell as in the state.
__global__ void __launch_bounds__(256) mlstm_chunk_scan_kernel(MlstmParams<bf16> p, ChunkView ws) {
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.y;
  const RaggedSeq seq = ragged_seq(p.seqs, b);
  if (!seq.live) return;
  const int mem = p.H * p.dk * p.dv / 4, total = mem + p.H * p.dk / 4;
  const int idx = blockIdx.x * 256 + threadIdx.x;
  if (idx >= total) return;
  const bool in_mem = idx < mem;
  const int h = in_mem ? idx / (p.dk * p.dv / 4) : (idx - mem) / (p.dk / 4);
  const bool first = in_mem && idx == h * (p.dk * p.dv / 4);       // this thread also keeps the head's running maximum
  const int chunks = (seq.rows + kC - 1) / kC;
  const size_t c0 = chunk_cell(seq, b, 0);
  float4* cell = reinterpret_cast<float4*>(ws.cells) + c0 * total + idx;
  const float2* sc = ws.scale + c0 * p.H + h;
  float* st = p.state + seq.slot * p.stride;
  float4* mine = reinterpret_cast<float4*>(st) + idx;
  float* m_state = st + static_cast<size_t>(p.H) * p.dk * (p.dv + 1) + h;
  float4 S = *mine;
  float m = *m_state * kLog2e;
  constexpr int kAhead = 4;
  float4 add[kAhead];
  float2 gate[kAhead];
  auto fetch = [&](int c, int i) {
    if (c < chunks) {
      add[i] = cell[static_cast<size_t>(c) * total];
      gate[i] = sc[static_cast<size_t>(c) * p.H];
    }
  };
#pragma unroll
  for (int i = 0; i < kAhead; ++i) fetch(i, i);
  for (int cb = 0; cb < chunks; cb += kAhead) {
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
      const int c = cb + i;
      if (c >= chunks) break;
      const float4 x = add[i];
      const float2 gt = gate[i];
      fetch(c + kAhead, i);
      if (in_mem) {
        uint4 u;
        split_pair(S.x, S.y, u.x, u.z);
        split_pair(S.z, S.w, u.y, u.w);
        *reinterpret_cast<uint4*>(cell + static_cast<size_t>(c) * total) = u;
      } else {
        cell[static_cast<size_t>(c) * total] = S;
      }
      if (first) ws.m_in[(c0 + c) * p.H + h] = m;
      const float m_new = fmaxf(gt.x + m, gt.y);
      const float keep = ex2_approx(gt.x + m - m_new), take = ex2_approx(gt.y - m_new);
      m = m_new;
      S = make_float4(fmaf(keep, S.x, take * x.x), fmaf(keep, S.y, take * x.y), fmaf(keep, S.z, take * x.z), fmaf(keep, S.w, take * x.w));
    }
  }
  *mine = S;
  // the running maximum is stored by mlstm_chunk_out: threads of other blocks of this launch may not have read it yet
  if (first) ws.m_in[(c0 + chunks) * p.H + h] = m;
}

// ---------------------------------------------------------------- 3. outputs
// grid (value tiles, chunks, H * B); the tiles of a head form a cluster and share the sums of squares of the outputs.
template <int NT>
__global__ void __launch_bounds__(kThr, NT == 1 ? 2 : 1) mlstm_chunk_out_kernel(MlstmParams<bf16> p, ChunkView ws, int tile_w) {
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ GateSmem gs;
  __shared__ float ssq[8][kC], tile_ss[kC], row_scale[kC], inv_den[kC];
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const TileGeom tg = tile_geom(p, tile_w);
  const RaggedSeq seq = ragged_seq(p.seqs, tg.b);
  const int t0 = blockIdx.y * kC;
  if (!seq.live || t0 >= seq.rows) return;  // uniform over the cluster
  const int dkp = key_pad(p.dk), ks = dkp + 8, vs = tile_w + 8, ss = 2 * tile_w + 8;
  bf16* q = reinterpret_cast<bf16*>(smem);           // [64][ks]
  bf16* k = q + kC * ks;                             // [64][ks]
  bf16* v = k + kC * ks;                             // [64][vs]
  bf16* ph = v + kC * vs;                            // gated scores hi / lo [64][kPStride]
  bf16* pl = ph + kC * kPStride;
  bf16* stage = pl + kC * kPStride;                  // [2][kStageRows][ss] entering state, [hi x 4 | lo x 4] per four columns
  float* n_in = reinterpret_cast<float*>(stage + 2 * kStageRows * ss);  // [dkp]
  const int n = min(kC, seq.rows - t0);
  const int qk = p.H * p.dk, vw = p.H * p.dv;
  const bf16* rows = p.proj + static_cast<size_t>(seq.row0 + t0) * p.ld;
  const size_t chunk = chunk_cell(seq, tg.b, blockIdx.y);
  const size_t per_chunk = static_cast<size_t>(p.H) * p.dk * (p.dv + 1);
  const float* cell = ws.cells + chunk * per_chunk;
  const bf16* S = reinterpret_cast<const bf16*>(cell + static_cast<size_t>(tg.h) * p.dk * p.dv + tg.c0);  // rows of 2 dv terms
  copy_tile(q, ks, rows + tg.h * p.dk, p.ld, kC, n, dkp / 8, p.dk / 8);
  copy_tile(k, ks, rows + qk + tg.h * p.dk, p.ld, kC, n, dkp / 8, p.dk / 8);
  copy_tile(v, vs, rows + 2 * qk + tg.h * p.dv + tg.c0, p.ld, kC, n, tg.width / 8, tg.width / 8);
  cp_async_commit();
  const int stages = (dkp + kStageRows - 1) / kStageRows;
  auto load_stage = [&](int i) {
    copy_tile(stage + (i & 1) * kStageRows * ss, ss, S + static_cast<size_t>(i) * kStageRows * 2 * p.dv, 2 * p.dv, kStageRows,
              p.dk - i * kStageRows, tg.width / 4, tg.width / 4);
    cp_async_commit();
  };
  load_stage(0);
  const float* nd = cell + static_cast<size_t>(p.H) * p.dk * p.dv + static_cast<size_t>(tg.h) * p.dk;
  for (int c = threadIdx.x; c < dkp; c += kThr) n_in[c] = c < p.dk ? nd[c] : 0.f;
  const float m_in = ws.m_in[chunk * p.H + tg.h];
  chunk_gates(p, gs, seq, tg.h, t0);
  cp_async_wait<1>();
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane >> 2, tig = lane & 3;
  const float q_scale = 1.f / sqrtf(static_cast<float>(p.dk));
  // ---- gated scores of the 16 x 16 blocks on and below the diagonal
  for (int i = warp; i < 10; i += 8) {
    const int I = i >= 6 ? 3 : i >= 3 ? 2 : i >= 1 ? 1 : 0, J = i - I * (I + 1) / 2;
    float acc[2][4] = {};
    for (int kk = 0; kk < dkp / 16; ++kk) {
      uint32_t a0, a1, a2, a3, b0, b1, b2, b3;
      ldsm_x4(smem_u32(q + (I * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ks + kk * 16 + (lane >> 4) * 8), a0, a1, a2, a3);
      ldsm_x4(smem_u32(k + (J * 16 + (lane & 7) + (lane >> 4) * 8) * ks + kk * 16 + ((lane >> 3) & 1) * 8), b0, b1, b2, b3);
      mma16816(acc[0], a0, a1, a2, a3, b0, b1);
      mma16816(acc[1], a0, a1, a2, a3, b2, b3);
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int t = I * 16 + g + r * 8, u = J * 16 + j * 8 + tig * 2;
        const float M = fmaxf(m_in, gs.top[t]);
        const float x = u <= t ? acc[j][2 * r] * q_scale * ex2_approx(gs.a[u] - M) : 0.f;
        const float y = u + 1 <= t ? acc[j][2 * r + 1] * q_scale * ex2_approx(gs.a[u + 1] - M) : 0.f;
        uint32_t hi, lo;
        split_pair(x, y, hi, lo);
        *reinterpret_cast<uint32_t*>(ph + t * kPStride + u) = hi;
        *reinterpret_cast<uint32_t*>(pl + t * kPStride + u) = lo;
      }
  }
  __syncthreads();
  {
    // ---- normaliser: four threads per token
    const int t = threadIdx.x >> 2, part = threadIdx.x & 3;
    const float M = fmaxf(m_in, gs.top[t]);
    const float rs = q_scale * ex2_approx(m_in - M);
    float dot = 0.f;
    for (int c = part * 2; c < dkp; c += 8) {
      const uint32_t qq = *reinterpret_cast<const uint32_t*>(q + t * ks + c);
      dot = fmaf(bf16_lo(qq), n_in[c], fmaf(bf16_hi(qq), n_in[c + 1], dot));
    }
    dot *= rs;
    for (int u = part * 2; u < (t & ~15) + 16; u += 8) {
      const uint32_t hi = *reinterpret_cast<const uint32_t*>(ph + t * kPStride + u), lo = *reinterpret_cast<const uint32_t*>(pl + t * kPStride + u);
      dot += bf16_lo(hi) + bf16_hi(hi) + bf16_lo(lo) + bf16_hi(lo);
    }
    dot += __shfl_xor_sync(0xffffffffu, dot, 1);
    dot += __shfl_xor_sync(0xffffffffu, dot, 2);
    if (part == 0) {
      row_scale[t] = rs;
      inv_den[t] = 1.f / (fmaxf(fabsf(dot), ex2_approx(-(gs.b[t] + M))) + kMlstmEps);
    }
  }
  // ---- entering state: [64 x dk] x [dk x 2 width]
  float acc2[2 * NT][4][4];
#pragma unroll
  for (int j = 0; j < 2 * NT; ++j)
#pragma unroll
    for (int m = 0; m < 4; ++m) acc2[j][m][0] = acc2[j][m][1] = acc2[j][m][2] = acc2[j][m][3] = 0.f;
  const int nt = tg.width / 8;                       // 8-column tiles of values; this warp's are warp * NT ...
  for (int i = 0; i < stages; ++i) {
    if (i + 1 < stages) load_stage(i + 1);
    else cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const bf16* sb = stage + (i & 1) * kStageRows * ss;
    if (warp * NT < nt) {
#pragma unroll
      for (int kk = 0; kk < kStageRows / 16; ++kk) {
        const int c = i * kStageRows + kk * 16;
        if (c >= dkp) break;
        uint32_t bf[2 * NT][2];
#pragma unroll
        for (int j = 0; j < NT; ++j)
          ldsm_x4_t(smem_u32(sb + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ss + (warp * NT + j) * 16 + (lane >> 4) * 8), bf[2 * j][0],
                    bf[2 * j][1], bf[2 * j + 1][0], bf[2 * j + 1][1]);
#pragma unroll
        for (int m = 0; m < 4; ++m) {
          uint32_t a0, a1, a2, a3;
          ldsm_x4(smem_u32(q + (m * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ks + c + (lane >> 4) * 8), a0, a1, a2, a3);
#pragma unroll
          for (int j = 0; j < 2 * NT; ++j) mma16816(acc2[j][m], a0, a1, a2, a3, bf[j][0], bf[j][1]);
        }
      }
    }
    __syncthreads();                                 // the stage is free for the load after the next
  }
  // columns 0-3 of a doubled tile are hi terms, 4-7 lo terms of the same four values; a tile of eight values is two doubled tiles
  float acc[NT][4][4];
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int m = 0; m < 4; ++m)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float x = acc2[2 * j][m][e] + __shfl_xor_sync(0xffffffffu, acc2[2 * j][m][e], 2);
        const float y = acc2[2 * j + 1][m][e] + __shfl_xor_sync(0xffffffffu, acc2[2 * j + 1][m][e], 2);
        acc[j][m][e] = (tig < 2 ? x : y) * row_scale[m * 16 + g + (e >> 1) * 8];
      }
  // ---- inside the chunk: scores x values (block rows see the block columns up to their own)
#pragma unroll
  for (int kk = 0; kk < 4; ++kk) {
    uint32_t vf[NT][2];
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int tile = min(warp * NT + j, nt - 1);
      uint32_t u2, u3;
      ldsm_x4_t(smem_u32(v + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * vs + tile * 8), vf[j][0], vf[j][1], u2, u3);
    }
#pragma unroll
    for (int m = kk; m < 4; ++m) {
      const int off = (m * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kPStride + kk * 16 + (lane >> 4) * 8;
      uint32_t a0, a1, a2, a3;
      ldsm_x4(smem_u32(ph + off), a0, a1, a2, a3);
#pragma unroll
      for (int j = 0; j < NT; ++j) mma16816(acc[j][m], a0, a1, a2, a3, vf[j][0], vf[j][1]);
      ldsm_x4(smem_u32(pl + off), a0, a1, a2, a3);
#pragma unroll
      for (int j = 0; j < NT; ++j) mma16816(acc[j][m], a0, a1, a2, a3, vf[j][0], vf[j][1]);
    }
  }
  // ---- normaliser, norm over the head's values, gate, store
  uint32_t gate[4][2][NT];
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = m * 16 + g + r * 8;
      const float d = inv_den[t];
      float sq = 0.f;
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        acc[j][m][2 * r] *= d;
        acc[j][m][2 * r + 1] *= d;
        const bool in = warp * NT + j < nt;
        if (in) sq += acc[j][m][2 * r] * acc[j][m][2 * r] + acc[j][m][2 * r + 1] * acc[j][m][2 * r + 1];
        gate[m][r][j] = in && t < n ? *reinterpret_cast<const uint32_t*>(rows + static_cast<size_t>(t) * p.ld + 2 * qk + vw + tg.h * p.dv + tg.c0 +
                                                                         (warp * NT + j) * 8 + tig * 2)
                                    : 0u;
      }
      sq += __shfl_xor_sync(0xffffffffu, sq, 1);
      sq += __shfl_xor_sync(0xffffffffu, sq, 2);
      if (tig == 0) ssq[warp][t] = sq;
    }
  __syncthreads();
  if (threadIdx.x < kC) {
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) tot += ssq[w][threadIdx.x];
    tile_ss[threadIdx.x] = tot;
  }
  if (gridDim.x > 1) {
    cluster_arrive_release();
    cluster_wait_acquire();
  } else {
    __syncthreads();
  }
  if (threadIdx.x < kC) {
    float tot = 0.f;
    if (gridDim.x > 1)
      for (int i = 0; i < static_cast<int>(gridDim.x); ++i) tot += cluster_f32(mapa_shared(smem_u32(&tile_ss[threadIdx.x]), i));
    else tot = tile_ss[threadIdx.x];
    ssq[0][threadIdx.x] = 1.f / sqrtf(tot / static_cast<float>(p.dv) + p.eps);
  }
  __syncthreads();
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = m * 16 + g + r * 8;
      if (t >= n) continue;
      const float inv = ssq[0][t];
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        if (warp * NT + j >= nt) continue;
        const int col = tg.h * p.dv + tg.c0 + (warp * NT + j) * 8 + tig * 2;
        const uint32_t gt = gate[m][r][j];
        const float2 w = *reinterpret_cast<const float2*>(p.norm_w + col);
        *reinterpret_cast<uint32_t*>(p.out + static_cast<size_t>(seq.row0 + t0 + t) * vw + col) =
            pack_bf16x2(acc[j][m][2 * r] * inv * w.x * sigmoid_fast(bf16_lo(gt)), acc[j][m][2 * r + 1] * inv * w.y * sigmoid_fast(bf16_hi(gt)));
      }
    }
  if (blockIdx.x == 0 && t0 + kC >= seq.rows && threadIdx.x == 0) {
    // the last chunk of the portion leaves the head's running maximum, which the scan put behind the chunks' own
    float* m_state = p.state + seq.slot * p.stride + static_cast<size_t>(p.H) * p.dk * (p.dv + 1) + tg.h;
    *m_state = ws.m_in[(chunk + 1) * p.H + tg.h] * (1.f / kLog2e);
  }
  if (gridDim.x > 1) {                               // nobody reads the sums of a CTA that has ended
    cluster_arrive_release();
    cluster_wait_acquire();
  }
}

bool mlstm_chunk_supported(int dk, int dv, int ld, long long stride) {
  return dk % 8 == 0 && dk <= kMaxKey && dv % 8 == 0 && dv <= kTileV * kMaxTiles && ld % 8 == 0 && stride % 4 == 0;
}

// Cells of the batch: one more per sequence than it has chunks (the running maximum that leaves the last one).
static long long chunk_cells(int rows, int batch) { return (rows + kC - 1) / kC + 2LL * batch; }

static long long align16(long long v) { return (v + 15) & ~15LL; }

long long mlstm_chunk_bytes(int H, int dk, int dv, int rows, int batch) {
  const long long cells = chunk_cells(rows, batch);
  return align16(cells * H * dk * (dv + 1) * 4) + align16(cells * H * 8) + align16(cells * H * 4);
}

template <int NT>
static cudaError_t launch_chunks(const MlstmParams<bf16>& p, int max_rows, const ChunkView& ws, int tiles, int tile_w, cudaStream_t stream) {
  const int ks = key_pad(p.dk) + 8, vs = tile_w + 8;
  const size_t smem_state = static_cast<size_t>(kC) * (2 * ks + vs) * sizeof(bf16);
  const size_t smem_out = (static_cast<size_t>(kC) * (2 * ks + vs + 2 * kPStride) + 2 * kStageRows * (2 * tile_w + 8)) * sizeof(bf16) +
                          key_pad(p.dk) * sizeof(float);
  static size_t configured[64] = {};
  int dev = 0;
  cudaError_t e = cudaGetDevice(&dev);
  if (e != cudaSuccess) return e;
  if (dev < 0 || dev >= 64) return cudaErrorInvalidDevice;
  if (configured[dev] < smem_out) {
    e = cudaFuncSetAttribute(mlstm_chunk_state_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem_out));
    if (e == cudaSuccess) e = cudaFuncSetAttribute(mlstm_chunk_out_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem_out));
    if (e != cudaSuccess) return e;
    configured[dev] = smem_out;
  }
  const dim3 grid(tiles, (max_rows + kC - 1) / kC, p.H * p.seqs.B);
  if (grid.y > 65535 || grid.z > 65535) return cudaErrorInvalidValue;
  e = launch_pdl(mlstm_chunk_state_kernel<NT>, grid, dim3(kThr), smem_state, stream, p, ws, tile_w);
  if (e != cudaSuccess) return e;
  const int quads = p.H * p.dk * (p.dv + 1) / 4;
  e = launch_pdl(mlstm_chunk_scan_kernel, dim3((quads + 255) / 256, p.seqs.B), dim3(256), 0, stream, p, ws);
  if (e != cudaSuccess) return e;
  cudaLaunchConfig_t lc = {};
  lc.gridDim = grid;
  lc.blockDim = dim3(kThr);
  lc.dynamicSmemBytes = smem_out;
  lc.stream = stream;
  cudaLaunchAttribute attr[2];
  int n = 0;
  if (pdl_enabled()) {
    attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[n].val.programmaticStreamSerializationAllowed = 1;
    ++n;
  }
  if (tiles > 1) {
    attr[n].id = cudaLaunchAttributeClusterDimension;
    attr[n].val.clusterDim.x = tiles;
    attr[n].val.clusterDim.y = 1;
    attr[n].val.clusterDim.z = 1;
    ++n;
  }
  lc.attrs = attr;
  lc.numAttrs = n;
  return cudaLaunchKernelEx(&lc, mlstm_chunk_out_kernel<NT>, p, ws, tile_w);
}

cudaError_t launch_mlstm_chunks(const MlstmParams<bf16>& p, int rows, int max_rows, void* scratch, cudaStream_t stream) {
  const long long cells = chunk_cells(rows, p.seqs.B);
  uint8_t* base = static_cast<uint8_t*>(scratch);
  ChunkView ws;
  ws.cells = reinterpret_cast<float*>(base);
  base += align16(cells * p.H * p.dk * (p.dv + 1) * 4);
  ws.scale = reinterpret_cast<float2*>(base);
  base += align16(cells * p.H * 8);
  ws.m_in = reinterpret_cast<float*>(base);
  const int tiles = (p.dv + kTileV - 1) / kTileV;
  const int tile_w = ((p.dv / 8 + tiles - 1) / tiles) * 8;
  return tile_w <= 64 ? launch_chunks<1>(p, max_rows, ws, tiles, tile_w, stream) : launch_chunks<2>(p, max_rows, ws, tiles, tile_w, stream);
}

}  // namespace eredu
