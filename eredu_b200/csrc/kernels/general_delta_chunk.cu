// Generalised delta rule over long portions, chunk-parallel on the tensor cores (recurrence and layout: general_delta.cu).
//
// Per head and chunk of 64 tokens, with l_t the log decay summed up to token t (l_{t-1}: up to the one before), l_end the whole chunk's,
// m = l_end / 2 and h = e^m per key channel, and rows
//   u~ = u e^{l_{t-1} - m},  r~ = r e^{l_t - m},  k~ = k e^{m - l_t},  b~ = a u e^{m - l_t},
// what token t finds under its key, p_t = u_t^T S_{t-1}, solves a unit lower-triangular system:
//   (I + A_ub) P = u~ (h S_in) + A_uk V       A_ub = u~ b~^T, A_uk = u~ k~^T below the diagonal
//   O = r~ (h S_in) + A_rk V - A_rb P         A_rk = r~ k~^T, A_rb = r~ b~^T up to the diagonal
//   S_out = h^2 S_in + h (k~^T V - b~^T P)
// With W = (I + A_ub)^{-1} u~ and X = (I + A_ub)^{-1} A_uk V everything that does not depend on S_in is known per chunk:
//   O = Y S_in + Z,  S_out = h^2 S_in + M S_in + N,
//   Y = (r~ - A_rb W) h,  Z = A_rk V - A_rb X,  M = -h (b~^T W) h,  N = h (k~^T V - b~^T X)
// so three launches do it, and only the second walks a sequence:
//   1. delta_chunk_kernel:  Y, Z, M, N, h^2 of every chunk. Scores by all warps (of u, later of r in their place), the inverses of the four
//      diagonal blocks by one each; a warp owns 16 columns of W or X from the substitution to what is stored, in registers.
//   2. delta_scan_kernel:   the state that enters every chunk, transposed; a few warps share 16 of its columns, the state stays in fp32
//      registers and meets the others of its group in shared memory once per chunk.
//   3. delta_out_kernel:    O, per-head norm, output gate.
// A decay step is at most e^-c, so the exponents stay within 32 c of zero: no blocks inside a chunk are needed.
//
// The products run on bf16 tensor cores without giving up 32-bit accuracy: every fp32 factor is split into two bf16 terms, hi + lo, and
// the cross terms are added (lo * lo is below 2^-16); values are bf16 to begin with. The diagonal part of a state update and the state
// itself are fp32.
#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/launch_count.h"
#include "../common/mma.cuh"
#include "../common/ptx.cuh"
#include "general_delta.h"

namespace eredu {

using bf16 = __nv_bfloat16;

constexpr int kC = 64;               // tokens of a chunk
constexpr int kChunkMinRows = 16;    // from this portion length on the chunk-parallel form takes over
constexpr float kMaxLogDecay = 2.f;  // 32 c log2(e) stays below 2^93

// What launch 1 leaves of one chunk and head, and launch 2 adds (`s`), head sizes padded to D.
template <int D>
struct DeltaCell {
  bf16 mh[D * D], ml[D * D];         // M [i][k]
  bf16 yh[kC * D], yl[kC * D];       // Y [t][i]
  bf16 sh[D * D], sl[D * D];         // entering state, transposed [j][i]
  float n[D * D];                    // N transposed [j][i]
  float z[kC * D];                   // Z [t][j]
  float h2[D];
};

// x = hi + lo with two bf16 terms, for a pair of values.
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(a, b);
  lo = pack_bf16x2(a - bf16_lo(hi), b - bf16_hi(hi));
}
// c += a b with both factors split, for N n-tiles
template <int N>
__device__ __forceinline__ void mma_split(float (&c)[N][4], const uint32_t (&ah)[4], const uint32_t (&al)[4], const uint32_t (&bh)[N][2], const uint32_t (&bl)[N][2]) {
#pragma unroll
  for (int n = 0; n < N; ++n) mma16816(c[n], ah[0], ah[1], ah[2], ah[3], bh[n][0], bh[n][1]);
#pragma unroll
  for (int n = 0; n < N; ++n) mma16816(c[n], ah[0], ah[1], ah[2], ah[3], bl[n][0], bl[n][1]);
#pragma unroll
  for (int n = 0; n < N; ++n) mma16816(c[n], al[0], al[1], al[2], al[3], bh[n][0], bh[n][1]);
}
// the same with a left factor that is exact in bf16
template <int N>
__device__ __forceinline__ void mma_left(float (&c)[N][4], const uint32_t (&f)[4], const uint32_t (&bh)[N][2], const uint32_t (&bl)[N][2]) {
#pragma unroll
  for (int n = 0; n < N; ++n) mma16816(c[n], f[0], f[1], f[2], f[3], bh[n][0], bh[n][1]);
#pragma unroll
  for (int n = 0; n < N; ++n) mma16816(c[n], f[0], f[1], f[2], f[3], bl[n][0], bl[n][1]);
}
__device__ __forceinline__ uint32_t ld32(const bf16* p) { return *reinterpret_cast<const uint32_t*>(p); }
__device__ __forceinline__ void st32(bf16* p, uint32_t v) { *reinterpret_cast<uint32_t*>(p) = v; }
// A fragment (16 rows x 16 k) of a row-major tile
__device__ __forceinline__ void frag_a(const bf16* tile, int stride, int lane, uint32_t (&f)[4]) {
  ldsm_x4(smem_u32(tile + ((lane & 7) + ((lane >> 3) & 1) * 8) * stride + (lane >> 4) * 8), f[0], f[1], f[2], f[3]);
}
// A fragment of the transpose of a row-major [16 k][16 rows] tile
__device__ __forceinline__ void frag_at(const bf16* tile, int stride, int lane, uint32_t (&f)[4]) {
  ldsm_x4_t(smem_u32(tile + ((lane & 7) + (lane >> 4) * 8) * stride + ((lane >> 3) & 1) * 8), f[0], f[1], f[2], f[3]);
}
// B fragments (16 k x 16 columns, two n-tiles) of a row-major [k][n] tile
__device__ __forceinline__ void frag_b(const bf16* tile, int stride, int lane, uint32_t (&f)[2][2]) {
  ldsm_x4_t(smem_u32(tile + ((lane & 7) + ((lane >> 3) & 1) * 8) * stride + (lane >> 4) * 8), f[0][0], f[0][1], f[1][0], f[1][1]);
}
// the same of a row-major [n][k] tile
__device__ __forceinline__ void frag_bt(const bf16* tile, int stride, int lane, uint32_t (&f)[2][2]) {
  ldsm_x4(smem_u32(tile + ((lane & 7) + (lane >> 4) * 8) * stride + ((lane >> 3) & 1) * 8), f[0][0], f[0][1], f[1][0], f[1][1]);
}
__device__ __forceinline__ int delta_chunk_id(const RaggedSeq& s, int b, int c) { return s.row0 / kC + b + c; }   // unique over the batch

constexpr int kBS = 24, kBlock = 16 * kBS;   // row stride and size of a 16 x 16 block of scores
__host__ __device__ constexpr int score_block(int I, int J) { return (I * (I + 1) / 2 + J) * kBlock; }

template <int D>
struct ChunkSmem {
  static constexpr int S = D + 8;    // row stride
  bf16 rh[kC * S], rl[kC * S], kh[kC * S], kl[kC * S], bh[kC * S], bl[kC * S], v[kC * S];
  bf16 uh[kC * S], ul[kC * S];       // first the decays' inputs, tanh hi and lo
  union {
    float dec[kC * S];               // log2 decay since the start of the token's block of 16, inclusive
    bf16 sc[4][10 * kBlock];         // scores up to the diagonal: against b hi, lo, against k hi, lo; of u first, then of r
  };
  float R[4 * D];                    // log2 decay at the starts of blocks 1, 2, 3 and at the end; later h in its first D
};

// Scores of one kind of row against b and k, in 16 x 16 blocks: below the diagonal (STRICT) or up to it.
template <int D, bool STRICT>
__device__ __forceinline__ void delta_scores(ChunkSmem<D>& s, const bf16* qh, const bf16* ql, int warp, int lane) {
  constexpr int S = ChunkSmem<D>::S;
  const int g = lane >> 2, tig = lane & 3;
  for (int i = warp; i < 20; i += 8) {
    const int blk = i >> 1, I = blk >= 6 ? 3 : blk >= 3 ? 2 : blk >= 1 ? 1 : 0, J = blk - I * (I + 1) / 2;
    const bool is_k = i & 1;
    const bf16 *xh = (is_k ? s.kh : s.bh) + J * 16 * S, *xl = (is_k ? s.kl : s.bl) + J * 16 * S;
    float acc[2][4] = {};
#pragma unroll
    for (int ks = 0; ks < D; ks += 16) {
      uint32_t ah[4], al[4], bh[2][2], bl[2][2];
      frag_a(qh + I * 16 * S + ks, S, lane, ah);
      frag_a(ql + I * 16 * S + ks, S, lane, al);
      frag_bt(xh + ks, S, lane, bh);
      frag_bt(xl + ks, S, lane, bl);
      mma_split(acc, ah, al, bh, bl);
    }
    bf16 *oh = s.sc[is_k ? 2 : 0] + blk * kBlock, *ol = s.sc[is_k ? 3 : 1] + blk * kBlock;
#pragma unroll
    for (int h = 0; h < 2; ++h)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int t = g + r * 8, c = h * 8 + tig * 2, last = I == J ? (STRICT ? t - 1 : t) : 16;   // last column that counts
        uint32_t hi, lo;
        split2(c <= last ? acc[h][2 * r] : 0.f, c + 1 <= last ? acc[h][2 * r + 1] : 0.f, hi, lo);
        st32(oh + t * kBS + c, hi);
        st32(ol + t * kBS + c, lo);
      }
  }
}

// ---------------------------------------------------------------- 1. chunks
template <int D>
__global__ void __launch_bounds__(256, D == 64 ? 2 : 1) delta_chunk_kernel(DeltaParams<bf16> p, DeltaCell<D>* __restrict__ cells) {
  using Sm = ChunkSmem<D>;
  constexpr int S = Sm::S;
  extern __shared__ __align__(16) uint8_t raw[];
  Sm& s = *reinterpret_cast<Sm*>(raw);
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int hd = blockIdx.y, b = blockIdx.z, t0 = blockIdx.x * kC;
  const RaggedSeq seq = ragged_seq(p.seqs, b);
  if (!seq.live || t0 >= seq.rows) return;                                // uniform
  const int n = min(kC, seq.rows - t0), dk = p.dk, dv = p.dv, rank = p.rank, rs = ((rank + 15) & ~15) + 8;
  const int qk = p.H * dk, vw = p.H * dv;
  const bf16* rows = p.proj + static_cast<size_t>(seq.row0 + t0) * p.ld;
  DeltaCell<D>& cell = cells[static_cast<size_t>(delta_chunk_id(seq, b, blockIdx.x)) * p.H + hd];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tig = lane & 3;
  bf16 *low_h = s.uh, *low_l = s.ul;

  // ---- rows of the chunk; rows behind the portion and channels behind the head size are zero
  constexpr int P = D / 8;
  for (int i = threadIdx.x; i < kC * P; i += 256) {
    const int t = i / P, c = (i % P) * 8;
    const bf16* src = rows + static_cast<size_t>(t) * p.ld;
    const int ok = t < n && c < dk ? 16 : 0, okv = t < n && c < dv ? 16 : 0;
    cp_async16(s.rh + t * S + c, ok ? src + hd * dk + c : rows, ok);
    cp_async16(s.kh + t * S + c, ok ? src + qk + hd * dk + c : rows, ok);
    cp_async16(s.bh + t * S + c, ok ? src + 2 * qk + 2 * vw + hd * dk + c : rows, ok);
    cp_async16(s.v + t * S + c, okv ? src + 2 * qk + hd * dv + c : rows, okv);
  }
  const int lp = (rs - 8) / 8;
  for (int i = threadIdx.x; i < kC * lp; i += 256) {
    const int t = i / lp, c = (i % lp) * 8;
    const int ok = t < n && c < rank ? 16 : 0;
    cp_async16(low_h + t * rs + c, ok ? rows + static_cast<size_t>(t) * p.ld + 3 * qk + 2 * vw + c : rows, ok);
  }
  cp_async_commit();
  cp_async_wait<0>();
  __syncthreads();
  for (int i = threadIdx.x; i < kC * lp * 4; i += 256) {
    const int t = i / (lp * 4), c = (i % (lp * 4)) * 2;
    const uint32_t x = ld32(low_h + t * rs + c);
    uint32_t hi, lo;
    split2(tanhf(bf16_lo(x)), tanhf(bf16_hi(x)), hi, lo);
    st32(low_h + t * rs + c, hi);
    st32(low_l + t * rs + c, lo);
  }
  __syncthreads();
  // ---- decays: a tile = one block of 16 tokens x 8 channels, summed along its tokens with shuffles
  for (int i = warp; i < 4 * (D / 8); i += 8) {
    const int blk = i & 3, c0 = (i >> 2) * 8;
    float acc[1][4] = {};
    const int ch = c0 + g;
    const float* w2 = p.w2 + static_cast<size_t>(hd * dk + min(ch, dk - 1)) * rank;
    for (int ks = 0; ks < rs - 8; ks += 16) {
      uint32_t ah[4], al[4], bh[1][2], bl[1][2];
      frag_a(low_h + blk * 16 * rs + ks, rs, lane, ah);
      frag_a(low_l + blk * 16 * rs + ks, rs, lane, al);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int k = ks + tig * 2 + e * 8;
        const bool in = k < rank && ch < dk;                              // rank is a multiple of eight
        const float2 w = in ? *reinterpret_cast<const float2*>(w2 + k) : make_float2(0.f, 0.f);
        split2(w.x, w.y, bh[0][e], bl[0][e]);
      }
      mma_split(acc, ah, al, bh, bl);
    }
    const int c = c0 + tig * 2;
    float d[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int cc = c + (e & 1), t = blk * 16 + g + (e >> 1) * 8;
      d[e] = cc < dk && t < n ? -p.log_decay * 1.4426950408889634f * sigmoid_fast(acc[0][e] + p.w0[hd * dk + cc]) : 0.f;
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
    *reinterpret_cast<float2*>(s.dec + (blk * 16 + g) * S + c) = make_float2(d[0], d[1]);
    *reinterpret_cast<float2*>(s.dec + (blk * 16 + g + 8) * S + c) = make_float2(d[2], d[3]);
  }
  __syncthreads();
  for (int c = threadIdx.x; c < D; c += 256) {
    float acc = 0.f;
    for (int blk = 0; blk < 4; ++blk) {
      acc += s.dec[(blk * 16 + 15) * S + c];
      s.R[blk * D + c] = acc;
    }
    cell.h2[c] = ex2_approx(acc);
  }
  __syncthreads();
  // ---- unit keys, removal rates and the four scaled rows, in place; a warp takes every eighth token
  {
    constexpr int Q = D / 64;                                             // channel pairs of a lane
    float mid[2 * Q], rb[2 * Q];
#pragma unroll
    for (int q = 0; q < Q; ++q) {
      const int c = lane * 2 + q * 64;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        mid[2 * q + e] = 0.5f * s.R[3 * D + c + e];
        rb[2 * q + e] = c + e < dk ? p.rate_b[hd * dk + c + e] : 0.f;
      }
    }
    for (int t = warp; t < kC; t += 8) {
      uint32_t kk[Q];
      float ss = 0.f;
#pragma unroll
      for (int q = 0; q < Q; ++q) {
        kk[q] = ld32(s.kh + t * S + lane * 2 + q * 64);
        ss += bf16_lo(kk[q]) * bf16_lo(kk[q]) + bf16_hi(kk[q]) * bf16_hi(kk[q]);
      }
      const float inv = 1.f / sqrtf(warp_sum_f32(ss) + kUnitEps);
#pragma unroll
      for (int q = 0; q < Q; ++q) {
        const int c = lane * 2 + q * 64, at = t * S + c;
        const uint32_t rr = ld32(s.rh + at), aa = ld32(s.bh + at);
        const float2 dec = *reinterpret_cast<const float2*>(s.dec + at);
        const float2 start = t < 16 ? make_float2(0.f, 0.f) : *reinterpret_cast<const float2*>(s.R + ((t >> 4) - 1) * D + c);
        const float2 before = (t & 15) == 0 ? make_float2(0.f, 0.f) : *reinterpret_cast<const float2*>(s.dec + at - S);
        const float l0 = start.x + dec.x - mid[2 * q], l1 = start.y + dec.y - mid[2 * q + 1];
        const float x0 = ex2_approx(start.x + before.x - mid[2 * q]), x1 = ex2_approx(start.y + before.y - mid[2 * q + 1]);
        const float e0 = ex2_approx(l0), e1 = ex2_approx(l1), i0 = ex2_approx(-l0), i1 = ex2_approx(-l1);
        const float k0 = bf16_lo(kk[q]), k1 = bf16_hi(kk[q]), u0 = k0 * inv, u1 = k1 * inv;
        const float a0 = sigmoid_fast(bf16_lo(aa) + rb[2 * q]), a1 = sigmoid_fast(bf16_hi(aa) + rb[2 * q + 1]);
        uint32_t hi, lo;
        split2(bf16_lo(rr) * e0, bf16_hi(rr) * e1, hi, lo);
        st32(s.rh + at, hi);
        st32(s.rl + at, lo);
        split2(k0 * i0, k1 * i1, hi, lo);
        st32(s.kh + at, hi);
        st32(s.kl + at, lo);
        split2(a0 * u0 * i0, a1 * u1 * i1, hi, lo);
        st32(s.bh + at, hi);
        st32(s.bl + at, lo);
        split2(u0 * x0, u1 * x1, hi, lo);
        st32(s.uh + at, hi);
        st32(s.ul + at, lo);
      }
    }
  }
  __syncthreads();
  for (int c = threadIdx.x; c < D; c += 256) s.R[c] = ex2_approx(0.5f * s.R[3 * D + c]);      // h
  delta_scores<D, true>(s, s.uh, s.ul, warp, lane);
  __syncthreads();
  // ---- inverses of the unit lower-triangular diagonal blocks, in their place: a lane forms one column by substitution
  if (warp < 4) {
    bf16 *lh = s.sc[0] + score_block(warp, warp), *ll = s.sc[1] + score_block(warp, warp);
    float x[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      float v = i == (lane & 15) ? 1.f : 0.f;
#pragma unroll
      for (int k = 0; k < i; ++k) v = fmaf(-(to_f32(lh[i * kBS + k]) + to_f32(ll[i * kBS + k])), x[k], v);
      x[i] = v;
    }
    __syncwarp();
    if (lane < 16)
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        const bf16 hi = __float2bfloat16(x[i]);
        lh[i * kBS + lane] = hi;
        ll[i * kBS + lane] = __float2bfloat16(x[i] - to_f32(hi));
      }
  }
  __syncthreads();
  // ---- 16 columns of W (from u~) or of X (from A_uk V), transposed: rows are columns, block I covers the tokens 16 I ..
  constexpr int G = D / 64;                                               // groups of columns a warp owns
  auto group_is_w = [&](int gi) { return G == 1 ? warp < 4 : gi == 0; };
  auto group_col = [&]() { return (G == 1 ? warp & 3 : warp) * 16; };
  const int c0 = group_col();
  uint32_t nh[G][4][4], nl[G][4][4];                                      // -W^T or -X^T as A fragments, hi and lo
#pragma unroll
  for (int gi = 0; gi < G; ++gi) {
    const bool is_w = group_is_w(gi);
#pragma unroll
    for (int I = 0; I < 4; ++I) {
      float acc[2][4] = {};
      if (is_w) {
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int at = (I * 16 + h * 8 + tig * 2 + (e & 1)) * S + c0 + g + (e >> 1) * 8;
            acc[h][e] = to_f32(s.uh[at]) + to_f32(s.ul[at]);
          }
      } else {
#pragma unroll
        for (int J = 0; J <= I; ++J) {
          uint32_t vf[4], bh[2][2], bl[2][2];
          frag_at(s.v + J * 16 * S + c0, S, lane, vf);
          frag_bt(s.sc[2] + score_block(I, J), kBS, lane, bh);
          frag_bt(s.sc[3] + score_block(I, J), kBS, lane, bl);
          mma_left(acc, vf, bh, bl);
        }
      }
#pragma unroll
      for (int J = 0; J < I; ++J) {
        uint32_t bh[2][2], bl[2][2];
        frag_bt(s.sc[0] + score_block(I, J), kBS, lane, bh);
        frag_bt(s.sc[1] + score_block(I, J), kBS, lane, bl);
        mma_split(acc, nh[gi][J], nl[gi][J], bh, bl);
      }
      uint32_t ah[4], al[4], ih[2][2], il[2][2];
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        split2(acc[h][0], acc[h][1], ah[2 * h], al[2 * h]);
        split2(acc[h][2], acc[h][3], ah[2 * h + 1], al[2 * h + 1]);
      }
      float x[2][4] = {};
      frag_bt(s.sc[0] + score_block(I, I), kBS, lane, ih);
      frag_bt(s.sc[1] + score_block(I, I), kBS, lane, il);
      mma_split(x, ah, al, ih, il);
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        split2(-x[h][0], -x[h][1], nh[gi][I][2 * h], nl[gi][I][2 * h]);
        split2(-x[h][2], -x[h][3], nh[gi][I][2 * h + 1], nl[gi][I][2 * h + 1]);
      }
    }
  }
  __syncthreads();                                                        // the scores of u are done with
  delta_scores<D, false>(s, s.rh, s.rl, warp, lane);
  __syncthreads();
#pragma unroll
  for (int gi = 0; gi < G; ++gi) {
    const bool is_w = group_is_w(gi);
    // as B fragments (k: tokens, n: the 16 columns) block J is {n[J][0], n[J][2]} and {n[J][1], n[J][3]}
    // ---- Y or Z: rows are tokens
#pragma unroll
    for (int I = 0; I < 4; ++I) {
      float acc[2][4];
#pragma unroll
      for (int h = 0; h < 2; ++h)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          float x = 0.f, y = 0.f;
          if (is_w) {
            const int at = (I * 16 + g + r * 8) * S + c0 + h * 8 + tig * 2;
            const uint32_t hi = ld32(s.rh + at), lo = ld32(s.rl + at);
            x = bf16_lo(hi) + bf16_lo(lo);
            y = bf16_hi(hi) + bf16_hi(lo);
          }
          acc[h][2 * r] = x;
          acc[h][2 * r + 1] = y;
        }
#pragma unroll
      for (int J = 0; J <= I; ++J) {
        uint32_t ah[4], al[4];
        frag_a(s.sc[0] + score_block(I, J), kBS, lane, ah);
        frag_a(s.sc[1] + score_block(I, J), kBS, lane, al);
        const uint32_t bh[2][2] = {{nh[gi][J][0], nh[gi][J][2]}, {nh[gi][J][1], nh[gi][J][3]}};
        const uint32_t bl[2][2] = {{nl[gi][J][0], nl[gi][J][2]}, {nl[gi][J][1], nl[gi][J][3]}};
        mma_split(acc, ah, al, bh, bl);
        if (!is_w) {
          uint32_t vb[2][2];
          frag_b(s.v + J * 16 * S + c0, S, lane, vb);
          frag_a(s.sc[2] + score_block(I, J), kBS, lane, ah);
          frag_a(s.sc[3] + score_block(I, J), kBS, lane, al);
#pragma unroll
          for (int h = 0; h < 2; ++h) mma16816(acc[h], ah[0], ah[1], ah[2], ah[3], vb[h][0], vb[h][1]);
#pragma unroll
          for (int h = 0; h < 2; ++h) mma16816(acc[h], al[0], al[1], al[2], al[3], vb[h][0], vb[h][1]);
        }
      }
#pragma unroll
      for (int h = 0; h < 2; ++h)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int c = c0 + h * 8 + tig * 2, at = (I * 16 + g + r * 8) * D + c;
          if (is_w) {
            uint32_t hi, lo;
            split2(acc[h][2 * r] * s.R[c], acc[h][2 * r + 1] * s.R[c + 1], hi, lo);
            st32(cell.yh + at, hi);
            st32(cell.yl + at, lo);
          } else {
            *reinterpret_cast<float2*>(cell.z + at) = make_float2(acc[h][2 * r], acc[h][2 * r + 1]);
          }
        }
    }
    // ---- M (rows are key channels) or N transposed (rows are this warp's value columns)
#pragma unroll 2
    for (int it = 0; it < D / 16; ++it) {
      float acc[2][4] = {};
#pragma unroll
      for (int J = 0; J < 4; ++J) {
        if (is_w) {
          uint32_t ah[4], al[4];
          frag_at(s.bh + J * 16 * S + it * 16, S, lane, ah);
          frag_at(s.bl + J * 16 * S + it * 16, S, lane, al);
          const uint32_t bh[2][2] = {{nh[gi][J][0], nh[gi][J][2]}, {nh[gi][J][1], nh[gi][J][3]}};
          const uint32_t bl[2][2] = {{nl[gi][J][0], nl[gi][J][2]}, {nl[gi][J][1], nl[gi][J][3]}};
          mma_split(acc, ah, al, bh, bl);
        } else {
          uint32_t vf[4], bh[2][2], bl[2][2];
          frag_b(s.bh + J * 16 * S + it * 16, S, lane, bh);
          frag_b(s.bl + J * 16 * S + it * 16, S, lane, bl);
          mma_split(acc, nh[gi][J], nl[gi][J], bh, bl);
          frag_at(s.v + J * 16 * S + c0, S, lane, vf);
          frag_b(s.kh + J * 16 * S + it * 16, S, lane, bh);
          frag_b(s.kl + J * 16 * S + it * 16, S, lane, bl);
          mma_left(acc, vf, bh, bl);
        }
      }
#pragma unroll
      for (int h = 0; h < 2; ++h)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          if (is_w) {
            const int row = it * 16 + g + r * 8, c = c0 + h * 8 + tig * 2;
            uint32_t hi, lo;
            split2(acc[h][2 * r] * s.R[row] * s.R[c], acc[h][2 * r + 1] * s.R[row] * s.R[c + 1], hi, lo);
            st32(cell.mh + row * D + c, hi);
            st32(cell.ml + row * D + c, lo);
          } else {
            const int c = it * 16 + h * 8 + tig * 2;
            *reinterpret_cast<float2*>(cell.n + (c0 + g + r * 8) * D + c) = make_float2(acc[h][2 * r] * s.R[c], acc[h][2 * r + 1] * s.R[c + 1]);
          }
        }
    }
  }
}

// ---------------------------------------------------------------- 2. entering states
// A CTA takes kTiles tiles of 16 value columns of one head; D / 16 warps share a tile, each with 16 key channels of the transposed state: a
// step of the walk is bound by the instructions of one warp.
template <int D>
struct ScanCfg {
  static constexpr int kParts = D / 16, kTiles = D == 64 ? 1 : 2, kWarps = kParts * kTiles, kThreads = 32 * kWarps;
  static constexpr int kStages = D == 64 ? 3 : 2, S = D + 8;
  static constexpr int kStage = 2 * D * S;                                // M hi, lo (elements)
  static constexpr int kSide = kTiles * 16 * S;                           // state hi or lo of the CTA's tiles
  static constexpr size_t kSmem = (static_cast<size_t>(kStages) * kStage + 4 * kSide) * sizeof(bf16);
};

template <int D>
__global__ void __launch_bounds__(ScanCfg<D>::kThreads) delta_scan_kernel(DeltaParams<bf16> p, DeltaCell<D>* __restrict__ cells) {
  using C = ScanCfg<D>;
  constexpr int S = C::S;
  extern __shared__ __align__(16) uint8_t raw[];
  bf16* ms = reinterpret_cast<bf16*>(raw);                                // [stage][hi, lo][D][S]
  bf16* ss = ms + C::kStages * C::kStage;                                 // [2][hi, lo][tiles * 16][S]
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int hd = blockIdx.y, b = blockIdx.z;
  const RaggedSeq seq = ragged_seq(p.seqs, b);
  if (!seq.live) return;                                                  // uniform
  const int chunks = (seq.rows + kC - 1) / kC;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tig = lane & 3;
  const int tile = warp / C::kParts, i0 = (warp % C::kParts) * 16, j0 = (blockIdx.x * C::kTiles + tile) * 16;
  DeltaCell<D>* cell = cells + static_cast<size_t>(delta_chunk_id(seq, b, 0)) * p.H + hd;
  float* st = p.state + (static_cast<size_t>(seq.slot) * p.H + hd) * p.dk * p.dv;
  float x[2][4];                                                          // S^T: rows j0 + g (+ 8), columns i0 + nt * 8 + tig * 2 (+ 1)
#pragma unroll
  for (int nt = 0; nt < 2; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int j = j0 + g + (e >> 1) * 8, i = i0 + nt * 8 + tig * 2 + (e & 1);
      x[nt][e] = i < p.dk && j < p.dv ? st[static_cast<size_t>(i) * p.dv + j] : 0.f;
    }
  auto fetch = [&](int c) {
    if (c < chunks) {
      const DeltaCell<D>& src = cell[static_cast<size_t>(c) * p.H];
      bf16* dst = ms + (c % C::kStages) * C::kStage;
      for (int i = threadIdx.x; i < 2 * D * (D / 8); i += C::kThreads) {
        const int lo = i / (D * (D / 8)), r = (i / (D / 8)) % D, q = (i % (D / 8)) * 8;
        cp_async16(dst + (lo * D + r) * S + q, (lo ? src.ml : src.mh) + r * D + q, 16);
      }
    }
    cp_async_commit();
  };
#pragma unroll
  for (int c = 0; c + 1 < C::kStages; ++c) fetch(c);
  float2 nn[2][2], hh[2];                                                 // what the chunk adds and h^2, in flight a chunk ahead
  auto ahead = [&](int c) {
    const DeltaCell<D>& src = cell[static_cast<size_t>(min(c, chunks - 1)) * p.H];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
      const int i = i0 + nt * 8 + tig * 2;
      hh[nt] = *reinterpret_cast<const float2*>(src.h2 + i);
#pragma unroll
      for (int r = 0; r < 2; ++r) nn[nt][r] = *reinterpret_cast<const float2*>(src.n + (j0 + g + r * 8) * D + i);
    }
  };
  // what launch 1 left has gone to memory by now: it comes back to L2 some chunks ahead, M by shares of the CTAs of the head
  constexpr int kAhead = 6;
  auto warm = [&](int c) {
    if (c >= chunks) return;
    const DeltaCell<D>& src = cell[static_cast<size_t>(c) * p.H];
    const uint32_t share = 4 * D * D / gridDim.x;
    bulk_prefetch_l2(reinterpret_cast<const char*>(src.mh) + blockIdx.x * share, share);
    bulk_prefetch_l2(src.n + blockIdx.x * C::kTiles * 16 * D, C::kTiles * 16 * D * sizeof(float));
    if (blockIdx.x == 0) bulk_prefetch_l2(src.h2, D * sizeof(float));
  };
  if (threadIdx.x == 0)
    for (int c = C::kStages - 1; c < kAhead; ++c) warm(c);
  ahead(0);
  for (int c = 0; c < chunks; ++c) {
    if (threadIdx.x == 0) warm(c + kAhead);
    DeltaCell<D>& now = cell[static_cast<size_t>(c) * p.H];
    bf16 *sh = ss + (c & 1) * 2 * C::kSide, *sl = sh + C::kSide;
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
      const int i = i0 + nt * 8 + tig * 2;
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        uint32_t hi, lo;
        split2(x[nt][2 * r], x[nt][2 * r + 1], hi, lo);
        const int at = (tile * 16 + g + r * 8) * S + i, out = (j0 + g + r * 8) * D + i;
        st32(sh + at, hi);
        st32(sl + at, lo);
        st32(now.sh + out, hi);
        st32(now.sl + out, lo);
      }
    }
    cp_async_wait<C::kStages - 2>();
    __syncthreads();                                                      // M of this chunk has landed, the state is in shared memory
    fetch(c + C::kStages - 1);                                            // into the stage of the chunk before, which everyone has left
    const bf16 *mh = ms + (c % C::kStages) * C::kStage + i0 * S, *ml = mh + D * S;
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) x[nt][e] = fmaf((e & 1) ? hh[nt].y : hh[nt].x, x[nt][e], (e & 1) ? nn[nt][e >> 1].y : nn[nt][e >> 1].x);
    ahead(c + 1);
#pragma unroll
    for (int ks = 0; ks < D; ks += 16) {
      uint32_t ah[4], al[4], bh[2][2], bl[2][2];
      frag_a(sh + tile * 16 * S + ks, S, lane, ah);
      frag_a(sl + tile * 16 * S + ks, S, lane, al);
      frag_bt(mh + ks, S, lane, bh);
      frag_bt(ml + ks, S, lane, bl);
      mma_split(x, ah, al, bh, bl);
    }
  }
#pragma unroll
  for (int nt = 0; nt < 2; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int j = j0 + g + (e >> 1) * 8, i = i0 + nt * 8 + tig * 2 + (e & 1);
      if (i < p.dk && j < p.dv) st[static_cast<size_t>(i) * p.dv + j] = x[nt][e];
    }
}

// ---------------------------------------------------------------- 3. outputs
// Eight warps: four blocks of 16 tokens x two halves of the value columns.
template <int D>
__global__ void __launch_bounds__(256) delta_out_kernel(DeltaParams<bf16> p, const DeltaCell<D>* __restrict__ cells) {
  constexpr int S = D + 8, NT = D / 16;                                   // n-tiles of a warp
  extern __shared__ __align__(16) uint8_t raw[];
  bf16 *yh = reinterpret_cast<bf16*>(raw), *yl = yh + kC * S, *sh = yl + kC * S, *sl = sh + D * S;
  __shared__ float ssq[2][kC];
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int hd = blockIdx.y, b = blockIdx.z, t0 = blockIdx.x * kC;
  const RaggedSeq seq = ragged_seq(p.seqs, b);
  if (!seq.live || t0 >= seq.rows) return;                                // uniform
  const DeltaCell<D>& cell = cells[static_cast<size_t>(delta_chunk_id(seq, b, blockIdx.x)) * p.H + hd];
  constexpr int P = D / 8;
  for (int i = threadIdx.x; i < kC * P; i += 256) {
    const int t = i / P, c = (i % P) * 8;
    cp_async16(yh + t * S + c, cell.yh + t * D + c, 16);
    cp_async16(yl + t * S + c, cell.yl + t * D + c, 16);
  }
  for (int i = threadIdx.x; i < D * P; i += 256) {
    const int r = i / P, c = (i % P) * 8;
    cp_async16(sh + r * S + c, cell.sh + r * D + c, 16);
    cp_async16(sl + r * S + c, cell.sl + r * D + c, 16);
  }
  cp_async_commit();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tig = lane & 3;
  const int I = warp >> 1, half = warp & 1, j0 = half * (D / 2);
  const int qk = p.H * p.dk, vw = p.H * p.dv;
  float acc[NT][4];
  uint32_t gate[NT][2];
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = I * 16 + g + r * 8, j = j0 + nt * 8 + tig * 2;
      const float2 z = *reinterpret_cast<const float2*>(cell.z + t * D + j);
      acc[nt][2 * r] = z.x;
      acc[nt][2 * r + 1] = z.y;
      gate[nt][r] = t0 + t < seq.rows && j < p.dv ? ld32(p.proj + static_cast<size_t>(seq.row0 + t0 + t) * p.ld + 2 * qk + vw + hd * p.dv + j) : 0u;
    }
  cp_async_wait<0>();
  __syncthreads();
#pragma unroll
  for (int ks = 0; ks < D; ks += 16) {
    uint32_t ah[4], al[4];
    frag_a(yh + I * 16 * S + ks, S, lane, ah);
    frag_a(yl + I * 16 * S + ks, S, lane, al);
#pragma unroll
    for (int n2 = 0; n2 < NT; n2 += 2) {
      uint32_t bh[2][2], bl[2][2];
      frag_bt(sh + (j0 + n2 * 8) * S + ks, S, lane, bh);
      frag_bt(sl + (j0 + n2 * 8) * S + ks, S, lane, bl);
      mma_split(*reinterpret_cast<float(*)[2][4]>(&acc[n2]), ah, al, bh, bl);
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    float q = 0.f;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) q += acc[nt][2 * r] * acc[nt][2 * r] + acc[nt][2 * r + 1] * acc[nt][2 * r + 1];
    q += __shfl_xor_sync(0xffffffffu, q, 1);
    q += __shfl_xor_sync(0xffffffffu, q, 2);
    if (tig == 0) ssq[half][I * 16 + g + r * 8] = q;
  }
  __syncthreads();
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int t = I * 16 + g + r * 8;
    if (t0 + t >= seq.rows) continue;
    const float inv = 1.f / sqrtf((ssq[0][t] + ssq[1][t]) / static_cast<float>(p.dv) + p.eps);
    bf16* out = p.out + static_cast<size_t>(seq.row0 + t0 + t) * vw + hd * p.dv;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
      const int j = j0 + nt * 8 + tig * 2;
      if (j >= p.dv) continue;
      const float2 w = *reinterpret_cast<const float2*>(p.norm_w + hd * p.dv + j);
      st32(out + j, pack_bf16x2(acc[nt][2 * r] * inv * w.x * sigmoid_fast(bf16_lo(gate[nt][r])), acc[nt][2 * r + 1] * inv * w.y * sigmoid_fast(bf16_hi(gate[nt][r]))));
    }
  }
}

static bool chunk_sizes(int dk, int dv) { return dk % 8 == 0 && dv % 8 == 0 && dk > 0 && dv > 0 && dk <= 128 && dv <= 128; }
static long long chunk_count(int rows, int batch) { return (rows + kC - 1) / kC + batch; }

// sizes padded to 64 or 128; the decays' inputs take the place of a tile
static int chunk_width(int dk, int dv, int rank) { return dk <= 64 && dv <= 64 && rank <= 64 ? 64 : 128; }

long long delta_chunk_bytes(int H, int dk, int dv, int rank, int rows, int batch, int max_rows) {
  if (max_rows < kChunkMinRows || !chunk_sizes(dk, dv)) return 0;
  const long long cell = chunk_width(dk, dv, rank) == 64 ? sizeof(DeltaCell<64>) : sizeof(DeltaCell<128>);
  return chunk_count(rows, batch) * H * cell;
}

template <int D>
static cudaError_t launch_chunks(const DeltaParams<bf16>& p, int max_rows, void* scratch, cudaStream_t stream) {
  constexpr size_t chunk_smem = sizeof(ChunkSmem<D>), out_smem = (2 * kC + 2 * D) * (D + 8) * sizeof(bf16);
  static_assert(chunk_smem <= 227 * 1024 && ScanCfg<D>::kSmem <= 227 * 1024, "shared memory");
  static bool configured[64] = {};
  int dev = 0;
  cudaError_t e = cudaGetDevice(&dev);
  if (e != cudaSuccess) return e;
  if (dev < 0 || dev >= 64) return cudaErrorInvalidDevice;
  if (!configured[dev]) {
    e = cudaFuncSetAttribute(delta_chunk_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(chunk_smem));
    if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_scan_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(ScanCfg<D>::kSmem));
    if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_out_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(out_smem));
    if (e != cudaSuccess) return e;
    configured[dev] = true;
  }
  DeltaCell<D>* cells = static_cast<DeltaCell<D>*>(scratch);
  const dim3 grid((max_rows + kC - 1) / kC, p.H, p.seqs.B);
  if (grid.y > 65535 || grid.z > 65535) return cudaErrorInvalidValue;
  e = launch_pdl(delta_chunk_kernel<D>, grid, dim3(256), chunk_smem, stream, p, cells);
  if (e != cudaSuccess) return e;
  e = launch_pdl(delta_scan_kernel<D>, dim3(D / 16 / ScanCfg<D>::kTiles, p.H, p.seqs.B), dim3(ScanCfg<D>::kThreads), ScanCfg<D>::kSmem, stream, p, cells);
  if (e != cudaSuccess) return e;
  eredu_count_launches(2);
  return launch_pdl(delta_out_kernel<D>, grid, dim3(256), out_smem, stream, p, static_cast<const DeltaCell<D>*>(cells));
}

bool delta_chunk_supported(const DeltaParams<bf16>& p) {
  return chunk_sizes(p.dk, p.dv) && p.rank % 8 == 0 && p.rank <= 128 && p.log_decay <= kMaxLogDecay && p.ld % 8 == 0 &&
         (reinterpret_cast<uintptr_t>(p.proj) & 15) == 0;
}

cudaError_t launch_delta_chunks(const DeltaParams<bf16>& p, int max_rows, void* scratch, cudaStream_t stream) {
  return chunk_width(p.dk, p.dv, p.rank) == 64 ? launch_chunks<64>(p, max_rows, scratch, stream) : launch_chunks<128>(p, max_rows, scratch, stream);
}

}  // namespace eredu
