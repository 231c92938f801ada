// Gated linear attention over long portions, chunk-parallel on the tensor cores (recurrence and layout: gla.cu).
//
// With b_t the log decay accumulated since the start of a chunk of 64 tokens,
//   o_t = (q_t e^{b_t})^T S_in + sum_{s <= t} (sum_i q_ti k_si e^{b_ti - b_si}) v_s
//   S_out = diag(e^{b_end}) S_in + sum_s (k_s e^{b_end - b_s}) v_s^T
// so three launches do all chunks of all sequences and heads at once, and only a scan over [dk, dv] matrices is sequential:
//   1. gla_chunk_state: what every chunk adds to the state (the sum over s above) and its decay e^{b_end}
//   2. gla_chunk_scan:  per matrix element, the state that enters every chunk (over the contributions, in place)
//   3. gla_chunk_out:   outputs, per-head norm and gate
// Every exponent is formed as a difference that is <= 0: a chunk is cut into four blocks of 16 tokens, scores between
// blocks are taken relative to the start of the later block, scores inside a block relative to half of the block's decay; a
// block whose decay is too strong for that (more than 2^-120 in 16 tokens) computes its scores pair by pair.
//
// The products run on bf16 tensor cores without giving up 32-bit accuracy: every fp32 factor (decayed queries and keys,
// scores, the state) is split into two bf16 terms, hi + lo, and the cross terms are added (the lo * lo term is below 2^-16);
// the values are bf16 to begin with.
#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/launch_count.h"
#include "../common/mma.cuh"
#include "../common/ptx.cuh"
#include "../common/ragged.cuh"
#include "gla.h"

namespace eredu {

using bf16 = __nv_bfloat16;

constexpr int kChunk = 64, kBlk = 16, kBlks = 4, kThreads = 256;
constexpr int kMaxDk = 128, kMaxDv = 256, kMaxRank = 64;
constexpr int kAStride = kChunk + 8;

// Shared memory of one chunk: rows of a padded width so that ldmatrix and fragment loads are free of bank conflicts.
struct ChunkSmem {
  bf16 *q, *k, *v, *ah, *al;   // q, k [64][ks]; v [64][vs]; scores hi / lo [64][kAStride]
  float *bl, *R;               // bl [64][ks]: log2 decay since the start of the token's block; R [5][dkp]: at block starts, end
  bf16 *low, *a2h, *a2l;       // inputs of the decays: low [64][rs], the expansion hi / lo [dkp][rs]
  int ks, vs, dkp, rs;
};

__host__ __device__ inline int chunk_dkp(int dk) { return (dk + 15) & ~15; }
__host__ __device__ inline size_t chunk_scores_bytes(int dk, int rank) {
  const size_t scores = 2 * kChunk * kAStride * sizeof(bf16);
  const size_t inputs = (2 * static_cast<size_t>(chunk_dkp(dk)) + kChunk) * (chunk_dkp(rank) + 8) * sizeof(bf16);
  return ((scores > inputs ? scores : inputs) + 15) & ~static_cast<size_t>(15);
}
__host__ __device__ inline size_t chunk_smem_bytes(int dk, int dv, int rank) {
  const size_t ks = chunk_dkp(dk) + 8;
  return kChunk * ks * (2 * sizeof(bf16) + sizeof(float)) + kChunk * static_cast<size_t>(dv + 8) * sizeof(bf16) +
         5 * chunk_dkp(dk) * sizeof(float) + chunk_scores_bytes(dk, rank);
}

__device__ __forceinline__ ChunkSmem chunk_smem(uint8_t* base, int dk, int dv, int rank) {
  ChunkSmem s;
  s.dkp = chunk_dkp(dk);
  s.ks = s.dkp + 8;
  s.vs = dv + 8;
  s.q = reinterpret_cast<bf16*>(base);
  s.k = s.q + kChunk * s.ks;
  s.v = s.k + kChunk * s.ks;
  s.bl = reinterpret_cast<float*>(s.v + kChunk * s.vs);
  s.R = s.bl + kChunk * s.ks;
  s.ah = reinterpret_cast<bf16*>(s.R + 5 * s.dkp);
  s.al = s.ah + kChunk * kAStride;
  s.rs = chunk_dkp(rank) + 8;
  s.low = s.ah;                            // dead before the scores are written
  s.a2h = s.low + kChunk * s.rs;
  s.a2l = s.a2h + s.dkp * s.rs;
  return s;
}

// x = hi + lo with two bf16 terms, for a pair of values.
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(a, b);
  lo = pack_bf16x2(a - bf16_lo(hi), b - bf16_hi(hi));
}

// log2(sigmoid(x)) = min(x, 0) log2(e) - log2(1 + t), t = e^-|x|. The logarithm of 1 + t keeps its relative accuracy for small t
// by the correction t / ((1 + t) - 1) (Goldberg, "What every computer scientist should know about floating-point arithmetic").
__device__ __forceinline__ float log2_sigmoid(float x) {
  const float y = x * 1.4426950408889634f;
  const float t = ex2_approx(-fabsf(y));
  const float u = 1.f + t;
  const float l = u == 1.f ? t * 1.4426950408889634f : __log2f(u) * __fdividef(t, u - 1.f);
  return fminf(y, 0.f) - l;
}

// Rows of the chunk and its decays. Tokens behind the portion: zero rows without decay.
template <bool WITH_Q>
__device__ __forceinline__ void load_chunk(const GlaParams<bf16>& p, const ChunkSmem& s, const RaggedSeq& seq, int h, int t0) {
  const int qk = p.H * p.dk, vw = p.H * p.dv;
  const int n = min(kChunk, seq.rows - t0);
  const bf16* rows = p.proj + static_cast<size_t>(seq.row0 + t0) * p.ld;
  const int kc = s.dkp / 8, kreal = p.dk / 8, vc = p.dv / 8;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rp = s.rs - 8;                                        // rank, padded to whole steps of the products
  // a warp takes every eighth row; half-warps take two rows at a time where a row has at most 16 pieces. Everything is in
  // flight at once.
  const int kper = kc <= 16 ? 2 : 1, kl = kc <= 16 ? lane & 15 : lane;
  for (int t = warp * kper + (kc <= 16 ? lane >> 4 : 0); t < kChunk; t += 8 * kper)
    for (int c = kl; c < kc; c += 32) {
      const int bytes = t < n && c < kreal ? 16 : 0;
      const bf16* src = bytes ? rows + static_cast<size_t>(t) * p.ld + h * p.dk + c * 8 : rows;
      if (WITH_Q) cp_async16(s.q + t * s.ks + c * 8, src, bytes);
      cp_async16(s.k + t * s.ks + c * 8, bytes ? src + qk : rows, bytes);
    }
  const int vper = vc <= 16 ? 2 : 1, vl = vc <= 16 ? lane & 15 : lane;
  for (int t = warp * vper + (vc <= 16 ? lane >> 4 : 0); t < kChunk; t += 8 * vper)
    for (int c = vl; c < vc; c += 32)
      cp_async16(s.v + t * s.vs + c * 8, t < n ? rows + static_cast<size_t>(t) * p.ld + 2 * qk + h * p.dv + c * 8 : rows, t < n ? 16 : 0);
  const int pieces = rp / 8;
  for (int i = threadIdx.x; i < kChunk * pieces; i += kThreads) {
    const int t = i / pieces, c = i % pieces;
    const int bytes = t < n && c * 8 < p.rank ? 16 : 0;
    cp_async16(s.low + t * s.rs + c * 8, bytes ? rows + static_cast<size_t>(t) * p.ld + 2 * qk + 2 * vw + c * 8 : rows, bytes);
  }
  cp_async_commit();
  const int quads = rp / 4;
  for (int i = threadIdx.x; i < s.dkp * quads; i += kThreads) {
    const int c = i / quads, j = (i % quads) * 4;
    const float4 w = c < p.dk && j < p.rank ? load4(p.a2 + (static_cast<size_t>(h) * p.dk + c) * p.rank + j) : make_float4(0.f, 0.f, 0.f, 0.f);
    uint2 hi, lo;
    split2(w.x, w.y, hi.x, lo.x);
    split2(w.z, w.w, hi.y, lo.y);
    *reinterpret_cast<uint2*>(s.a2h + c * s.rs + j) = hi;
    *reinterpret_cast<uint2*>(s.a2l + c * s.rs + j) = lo;
  }
  cp_async_wait<0>();
  __syncthreads();
  // z = low a2^T + bias on the tensor cores, one tile = one block of 16 tokens x 8 channels; the decays are summed along the
  // tokens of the tile with shuffles (lane group g holds the rows g and g + 8)
  const int g = lane >> 2, tig = lane & 3;
  for (int i = warp; i < kBlks * (s.dkp / 8); i += 8) {
    const int blk = i & (kBlks - 1), c0 = (i / kBlks) * 8;
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int ks = 0; ks < rp; ks += 16) {
      const bf16* lo = s.low + (blk * kBlk + g) * s.rs + ks + tig * 2;
      const uint32_t a0 = *reinterpret_cast<const uint32_t*>(lo), a1 = *reinterpret_cast<const uint32_t*>(lo + 8 * s.rs);
      const uint32_t a2 = *reinterpret_cast<const uint32_t*>(lo + 8), a3 = *reinterpret_cast<const uint32_t*>(lo + 8 * s.rs + 8);
      const int off = (c0 + g) * s.rs + ks + tig * 2;
      mma16816(acc, a0, a1, a2, a3, *reinterpret_cast<const uint32_t*>(s.a2h + off), *reinterpret_cast<const uint32_t*>(s.a2h + off + 8));
      mma16816(acc, a0, a1, a2, a3, *reinterpret_cast<const uint32_t*>(s.a2l + off), *reinterpret_cast<const uint32_t*>(s.a2l + off + 8));
    }
    const int c = c0 + tig * 2;
    float d[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int ch = c + (e & 1), t = blk * kBlk + g + (e >> 1) * 8;
      d[e] = ch < p.dk && t < n ? log2_sigmoid(acc[e] + p.a2_b[h * p.dk + ch]) * p.inv_tau : 0.f;
    }
#pragma unroll
    for (int o = 4; o < 32; o <<= 1)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float up = __shfl_up_sync(0xffffffffu, d[e], o);
        if (lane >= o) d[e] += up;
      }
    d[2] += __shfl_sync(0xffffffffu, d[0], 28 + tig);
    d[3] += __shfl_sync(0xffffffffu, d[1], 28 + tig);
    *reinterpret_cast<float2*>(s.bl + (blk * kBlk + g) * s.ks + c) = make_float2(d[0], d[1]);
    *reinterpret_cast<float2*>(s.bl + (blk * kBlk + g + 8) * s.ks + c) = make_float2(d[2], d[3]);
  }
  __syncthreads();
  for (int c = threadIdx.x; c < s.dkp; c += kThreads) {
    float acc = 0.f;
    for (int blk = 0; blk < kBlks; ++blk) {
      s.R[blk * s.dkp + c] = acc;
      acc += s.bl[(blk * kBlk + kBlk - 1) * s.ks + c];
    }
    s.R[kBlks * s.dkp + c] = acc;
  }
  __syncthreads();
}

__device__ __forceinline__ int chunk_id(const RaggedSeq& s, int b, int c) { return s.row0 / kChunk + b + c; }  // unique over the batch

// ---------------------------------------------------------------- 1. contributions of the chunks
template <int NT>
__global__ void __launch_bounds__(kThreads, NT <= 2 ? 2 : 1) gla_chunk_state_kernel(GlaParams<bf16> p, float* __restrict__ ws, float* __restrict__ decay) {
  extern __shared__ __align__(16) uint8_t smem[];
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int h = blockIdx.y, b = blockIdx.z;
  const RaggedSeq seq = ragged_seq(p.seqs, b);
  if (!seq.live || static_cast<int>(blockIdx.x) * kChunk >= seq.rows) return;  // uniform
  const ChunkSmem s = chunk_smem(smem, p.dk, p.dv, p.rank);
  load_chunk<false>(p, s, seq, h, blockIdx.x * kChunk);
  const size_t cell = static_cast<size_t>(chunk_id(seq, b, blockIdx.x)) * p.H + h;
  // k e^{b_end - b_s}: hi over the keys, lo in the place of the queries
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int c = lane * 2; c < s.dkp; c += 64) {
    const float2 end = *reinterpret_cast<const float2*>(s.R + kBlks * s.dkp + c);
#pragma unroll
    for (int i = 0; i < kChunk / 8; ++i) {                         // this warp's rows: two of every block
      const int t = warp + 8 * i;
      const uint32_t kk = *reinterpret_cast<const uint32_t*>(s.k + t * s.ks + c);
      const float2 r0 = *reinterpret_cast<const float2*>(s.R + (i >> 1) * s.dkp + c);
      const float2 bl = *reinterpret_cast<const float2*>(s.bl + t * s.ks + c);
      uint32_t hi, lo;
      split2(bf16_lo(kk) * ex2_approx(end.x - r0.x - bl.x), bf16_hi(kk) * ex2_approx(end.y - r0.y - bl.y), hi, lo);
      *reinterpret_cast<uint32_t*>(s.k + t * s.ks + c) = hi;
      *reinterpret_cast<uint32_t*>(s.q + t * s.ks + c) = lo;
    }
  }
  for (int c = threadIdx.x; c < p.dk; c += kThreads) decay[cell * p.dk + c] = ex2_approx(s.R[kBlks * s.dkp + c]);
  __syncthreads();
  const int g = lane >> 2, tig = lane & 3;
  const int nt = p.dv / 8;
  uint32_t vf[NT][8];
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    const int tile = min(warp + 8 * j, nt - 1);
#pragma unroll
    for (int half = 0; half < 2; ++half)
      ldsm_x4_t(smem_u32(s.v + (half * 32 + (lane & 7) + ((lane >> 3) & 1) * 8 + (lane >> 4) * 16) * s.vs + tile * 8),
                vf[j][4 * half], vf[j][4 * half + 1], vf[j][4 * half + 2], vf[j][4 * half + 3]);
  }
  float* out = ws + cell * p.dk * p.dv;
  for (int mt = 0; mt < s.dkp / 16; ++mt) {
    float acc[NT][4];
#pragma unroll
    for (int j = 0; j < NT; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      const int off = (ks * 16 + (lane & 7) + (lane >> 4) * 8) * s.ks + mt * 16 + ((lane >> 3) & 1) * 8;
      uint32_t a0, a1, a2, a3;
      ldsm_x4_t(smem_u32(s.k + off), a0, a1, a2, a3);
#pragma unroll
      for (int j = 0; j < NT; ++j) mma16816(acc[j], a0, a1, a2, a3, vf[j][2 * ks], vf[j][2 * ks + 1]);
      ldsm_x4_t(smem_u32(s.q + off), a0, a1, a2, a3);
#pragma unroll
      for (int j = 0; j < NT; ++j) mma16816(acc[j], a0, a1, a2, a3, vf[j][2 * ks], vf[j][2 * ks + 1]);
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
__global__ void __launch_bounds__(256) gla_chunk_scan_kernel(GlaParams<bf16> p, float* __restrict__ ws, const float* __restrict__ decay) {
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.y;
  const RaggedSeq seq = ragged_seq(p.seqs, b);
  if (!seq.live) return;
  const int per_head = p.dk * p.dv / 4;
  const int idx = blockIdx.x * 256 + threadIdx.x;
  if (idx >= p.H * per_head) return;
  const int row = idx / (p.dv / 4);                               // h * dk + channel
  const int chunks = (seq.rows + kChunk - 1) / kChunk;
  const size_t step = static_cast<size_t>(p.H) * per_head, dstep = static_cast<size_t>(p.H) * p.dk;
  float4* cell = reinterpret_cast<float4*>(ws) + static_cast<size_t>(chunk_id(seq, b, 0)) * step + idx;
  const float* d = decay + static_cast<size_t>(chunk_id(seq, b, 0)) * dstep + row;
  float4* st = reinterpret_cast<float4*>(p.state) + static_cast<size_t>(seq.slot) * step + idx;
  float4 S = *st;
  constexpr int kAhead = 4;
  float4 add[kAhead];
  float dec[kAhead];
  auto fetch = [&](int c, int i) {
    if (c < chunks) {
      add[i] = cell[c * step];
      dec[i] = d[c * dstep];
    }
  };
#pragma unroll
  for (int i = 0; i < kAhead; ++i) fetch(i, i);
  for (int c0 = 0; c0 < chunks; c0 += kAhead) {
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
      if (c0 + i >= chunks) break;
      const float4 x = add[i];
      const float e = dec[i];
      fetch(c0 + i + kAhead, i);
      cell[(c0 + i) * step] = S;
      S = make_float4(fmaf(e, S.x, x.x), fmaf(e, S.y, x.y), fmaf(e, S.z, x.z), fmaf(e, S.w, x.w));
    }
  }
  *st = S;
}

// ---------------------------------------------------------------- 3. outputs
// Scores of block row I against block column J (16 x 16) by one warp, split into the two bf16 score tiles.
__device__ __forceinline__ void score_block(const ChunkSmem& s, int I, int J, float q_scale, int lane) {
  const int g = lane >> 2, tig = lane & 3;
  const bool diag = I == J;
  const float* tot = s.bl + (I * kBlk + kBlk - 1) * s.ks;          // decay over the whole block
  if (diag) {
    bool strong = false;
    for (int c = lane; c < s.dkp; c += 32) strong |= tot[c] < -120.f;
    if (__any_sync(0xffffffffu, strong)) {
      for (int e = lane; e < kBlk * kBlk; e += 32) {
        const int t = I * kBlk + e / kBlk, u = I * kBlk + e % kBlk;
        float a = 0.f;
        if (u <= t)
          for (int c = 0; c < s.dkp; ++c)
            a = fmaf(to_f32(s.q[t * s.ks + c]) * to_f32(s.k[u * s.ks + c]), ex2_approx(s.bl[t * s.ks + c] - s.bl[u * s.ks + c]), a);
        a *= q_scale;
        const bf16 hi = __float2bfloat16(a);
        s.ah[t * kAStride + u] = hi;
        s.al[t * kAStride + u] = __float2bfloat16(a - to_f32(hi));
      }
      return;
    }
  }
  float acc[2][4] = {};
  for (int ks = 0; ks < s.dkp / 16; ++ks) {
    uint32_t ah[4], al[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {                                   // (row g, k low), (g + 8, low), (g, high), (g + 8, high)
      const int t = I * kBlk + g + (i & 1) * 8, c = ks * 16 + tig * 2 + (i >> 1) * 8;
      const uint32_t q = *reinterpret_cast<const uint32_t*>(s.q + t * s.ks + c);
      const float2 bl = *reinterpret_cast<const float2*>(s.bl + t * s.ks + c);
      const float r0 = diag ? 0.5f * tot[c] : 0.f, r1 = diag ? 0.5f * tot[c + 1] : 0.f;
      split2(bf16_lo(q) * q_scale * ex2_approx(bl.x - r0), bf16_hi(q) * q_scale * ex2_approx(bl.y - r1), ah[i], al[i]);
    }
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int u = J * kBlk + j * 8 + g;
      uint32_t bh[2], bo[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int c = ks * 16 + tig * 2 + i * 8;
        const uint32_t k = *reinterpret_cast<const uint32_t*>(s.k + u * s.ks + c);
        const float2 bl = *reinterpret_cast<const float2*>(s.bl + u * s.ks + c);
        const float r0 = diag ? 0.5f * tot[c] : s.R[I * s.dkp + c] - s.R[J * s.dkp + c];
        const float r1 = diag ? 0.5f * tot[c + 1] : s.R[I * s.dkp + c + 1] - s.R[J * s.dkp + c + 1];
        split2(bf16_lo(k) * ex2_approx(r0 - bl.x), bf16_hi(k) * ex2_approx(r1 - bl.y), bh[i], bo[i]);
      }
      mma16816(acc[j], ah[0], ah[1], ah[2], ah[3], bh[0], bh[1]);
      mma16816(acc[j], ah[0], ah[1], ah[2], ah[3], bo[0], bo[1]);
      mma16816(acc[j], al[0], al[1], al[2], al[3], bh[0], bh[1]);
    }
  }
#pragma unroll
  for (int j = 0; j < 2; ++j)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = g + r * 8, u = j * 8 + tig * 2;
      const float x = !diag || u <= t ? acc[j][2 * r] : 0.f, y = !diag || u + 1 <= t ? acc[j][2 * r + 1] : 0.f;
      uint32_t hi, lo;
      split2(x, y, hi, lo);
      *reinterpret_cast<uint32_t*>(s.ah + (I * kBlk + t) * kAStride + J * kBlk + u) = hi;
      *reinterpret_cast<uint32_t*>(s.al + (I * kBlk + t) * kAStride + J * kBlk + u) = lo;
    }
}

template <int NT>
__global__ void __launch_bounds__(kThreads, NT <= 2 ? 2 : 1) gla_chunk_out_kernel(GlaParams<bf16> p, const float* __restrict__ ws) {
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float ssq[8][kChunk];
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int h = blockIdx.y, b = blockIdx.z;
  const RaggedSeq seq = ragged_seq(p.seqs, b);
  const int t0 = blockIdx.x * kChunk;
  if (!seq.live || t0 >= seq.rows) return;  // uniform
  const ChunkSmem s = chunk_smem(smem, p.dk, p.dv, p.rank);
  const float* S = ws + (static_cast<size_t>(chunk_id(seq, b, blockIdx.x)) * p.H + h) * p.dk * p.dv;
  if (threadIdx.x < 32)                                           // on its way to L2 while the scores are formed
    for (int r = threadIdx.x; r < p.dk; r += 32) bulk_prefetch_l2(S + static_cast<size_t>(r) * p.dv, p.dv * 4);
  load_chunk<true>(p, s, seq, h, t0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane >> 2, tig = lane & 3;
  const float q_scale = 1.f / sqrtf(static_cast<float>(p.dk));
  for (int i = warp; i < kBlks * (kBlks + 1) / 2; i += 8) {
    const int I = i >= 6 ? 3 : i >= 3 ? 2 : i >= 1 ? 1 : 0;
    score_block(s, I, i - I * (I + 1) / 2, q_scale, lane);
  }
  __syncthreads();
  // q e^{b_t} / sqrt(dk): hi in the place of the keys, lo over the queries
  for (int c = lane * 2; c < s.dkp; c += 64) {
#pragma unroll
    for (int i = 0; i < kChunk / 8; ++i) {
      const int t = warp + 8 * i;
      const uint32_t q = *reinterpret_cast<const uint32_t*>(s.q + t * s.ks + c);
      const float2 bl = *reinterpret_cast<const float2*>(s.bl + t * s.ks + c);
      const float2 r = *reinterpret_cast<const float2*>(s.R + (i >> 1) * s.dkp + c);
      uint32_t hi, lo;
      split2(bf16_lo(q) * q_scale * ex2_approx(r.x + bl.x), bf16_hi(q) * q_scale * ex2_approx(r.y + bl.y), hi, lo);
      *reinterpret_cast<uint32_t*>(s.k + t * s.ks + c) = hi;
      *reinterpret_cast<uint32_t*>(s.q + t * s.ks + c) = lo;
    }
  }
  __syncthreads();
  const int nt = p.dv / 8;
  float acc[NT][4][4];
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int m = 0; m < 4; ++m) acc[j][m][0] = acc[j][m][1] = acc[j][m][2] = acc[j][m][3] = 0.f;
  // ---- entering state: [64 x dk] x [dk x dv]; its fragments come straight from global memory, once per CTA
#pragma unroll 4
  for (int ks = 0; ks < s.dkp / 16; ++ks) {
    uint32_t bh[NT][2], bo[NT][2];
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int n = min(warp + 8 * j, nt - 1) * 8 + g;
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int r = ks * 16 + tig * 2 + i * 8;
        const float x = r < p.dk ? S[static_cast<size_t>(r) * p.dv + n] : 0.f;
        const float y = r + 1 < p.dk ? S[static_cast<size_t>(r + 1) * p.dv + n] : 0.f;
        split2(x, y, bh[j][i], bo[j][i]);
      }
    }
#pragma unroll
    for (int m = 0; m < 4; ++m) {
      const int off = (m * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * s.ks + ks * 16 + (lane >> 4) * 8;
      uint32_t a0, a1, a2, a3, l0, l1, l2, l3;
      ldsm_x4(smem_u32(s.k + off), a0, a1, a2, a3);
      ldsm_x4(smem_u32(s.q + off), l0, l1, l2, l3);
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        mma16816(acc[j][m], a0, a1, a2, a3, bh[j][0], bh[j][1]);
        mma16816(acc[j][m], a0, a1, a2, a3, bo[j][0], bo[j][1]);
        mma16816(acc[j][m], l0, l1, l2, l3, bh[j][0], bh[j][1]);
      }
    }
  }
  // ---- inside the chunk: scores x values (block rows see the block columns up to their own)
#pragma unroll
  for (int ks = 0; ks < kBlks; ++ks) {
    uint32_t vf[NT][2];
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int tile = min(warp + 8 * j, nt - 1);
      uint32_t u2, u3;
      ldsm_x4_t(smem_u32(s.v + (ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * s.vs + tile * 8), vf[j][0], vf[j][1], u2, u3);
    }
#pragma unroll
    for (int m = ks; m < kBlks; ++m) {
      const int off = (m * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kAStride + ks * 16 + (lane >> 4) * 8;
      uint32_t a0, a1, a2, a3;
      ldsm_x4(smem_u32(s.ah + off), a0, a1, a2, a3);
#pragma unroll
      for (int j = 0; j < NT; ++j) mma16816(acc[j][m], a0, a1, a2, a3, vf[j][0], vf[j][1]);
      ldsm_x4(smem_u32(s.al + off), a0, a1, a2, a3);
#pragma unroll
      for (int j = 0; j < NT; ++j) mma16816(acc[j][m], a0, a1, a2, a3, vf[j][0], vf[j][1]);
    }
  }
  // ---- norm over the head's values, gate, store
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float ss = 0.f;
#pragma unroll
      for (int j = 0; j < NT; ++j)
        if (warp + 8 * j < nt) ss += acc[j][m][2 * r] * acc[j][m][2 * r] + acc[j][m][2 * r + 1] * acc[j][m][2 * r + 1];
      ss += __shfl_xor_sync(0xffffffffu, ss, 1);
      ss += __shfl_xor_sync(0xffffffffu, ss, 2);
      if (tig == 0) ssq[warp][m * 16 + g + r * 8] = ss;
    }
  const int qk = p.H * p.dk, vw = p.H * p.dv;
  uint32_t gate[4][2][NT];
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = t0 + m * 16 + g + r * 8;
#pragma unroll
      for (int j = 0; j < NT; ++j)
        gate[m][r][j] = t < seq.rows && warp + 8 * j < nt
                            ? *reinterpret_cast<const uint32_t*>(p.proj + static_cast<size_t>(seq.row0 + t) * p.ld + 2 * qk + vw + h * p.dv +
                                                                 (warp + 8 * j) * 8 + tig * 2)
                            : 0u;
    }
  __syncthreads();
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = m * 16 + g + r * 8;
      if (t0 + t >= seq.rows) continue;
      float tot = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) tot += ssq[w][t];
      const float inv = 1.f / sqrtf(tot / static_cast<float>(p.dv) + p.eps);
      const size_t row = static_cast<size_t>(seq.row0 + t0 + t);
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        if (warp + 8 * j >= nt) continue;
        const int n = (warp + 8 * j) * 8 + tig * 2;
        const uint32_t gt = gate[m][r][j];
        const float2 w = *reinterpret_cast<const float2*>(p.norm_w + n);
        *reinterpret_cast<uint32_t*>(p.out + row * vw + h * p.dv + n) =
            pack_bf16x2(acc[j][m][2 * r] * inv * w.x * silu_fast(bf16_lo(gt)), acc[j][m][2 * r + 1] * inv * w.y * silu_fast(bf16_hi(gt)));
      }
    }
}

bool gla_chunk_supported(const GlaParams<bf16>& p) {
  return p.dk % 8 == 0 && p.dk <= kMaxDk && p.dv % 8 == 0 && p.dv <= kMaxDv && p.rank <= kMaxRank && p.rank % 8 == 0 && p.ld % 8 == 0 &&
         (reinterpret_cast<uintptr_t>(p.proj) & 15) == 0;
}

long long gla_chunk_count(int rows, int batch) { return (rows + kChunk - 1) / kChunk + batch; }

template <int NT>
static cudaError_t launch_chunks(const GlaParams<bf16>& p, int max_rows, float* ws, float* decay, cudaStream_t stream) {
  const size_t smem = chunk_smem_bytes(p.dk, p.dv, p.rank);
  static size_t configured[64] = {};
  int dev = 0;
  cudaError_t e = cudaGetDevice(&dev);
  if (e != cudaSuccess) return e;
  if (dev < 0 || dev >= 64) return cudaErrorInvalidDevice;
  if (configured[dev] < smem) {
    e = cudaFuncSetAttribute(gla_chunk_state_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e == cudaSuccess) e = cudaFuncSetAttribute(gla_chunk_out_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return e;
    configured[dev] = smem;
  }
  const dim3 grid((max_rows + kChunk - 1) / kChunk, p.H, p.seqs.B);
  e = launch_pdl(gla_chunk_state_kernel<NT>, grid, dim3(kThreads), smem, stream, p, ws, decay);
  if (e != cudaSuccess) return e;
  e = launch_pdl(gla_chunk_scan_kernel, dim3((p.H * p.dk * p.dv / 4 + 255) / 256, p.seqs.B), dim3(256), 0, stream, p, ws,
                 static_cast<const float*>(decay));
  if (e != cudaSuccess) return e;
  return launch_pdl(gla_chunk_out_kernel<NT>, grid, dim3(kThreads), smem, stream, p, static_cast<const float*>(ws));
}

cudaError_t launch_gla_chunks(const GlaParams<bf16>& p, int max_rows, float* ws, float* decay, cudaStream_t stream) {
  switch ((p.dv / 8 + 7) / 8) {
    case 1: return launch_chunks<1>(p, max_rows, ws, decay, stream);
    case 2: return launch_chunks<2>(p, max_rows, ws, decay, stream);
    default: return launch_chunks<4>(p, max_rows, ws, decay, stream);
  }
}

}  // namespace eredu
