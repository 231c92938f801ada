// Prefill attention on the 5th-generation tensor cores: S = Q K^T and O += P V are tcgen05.mma with the accumulators in
// tensor memory, K / V pages arrive by TMA straight from the paged cache.
//
// One CTA = 256 query rows (two tiles of 128, "a" and "b") of one (sequence, query head); keys are walked in tiles of 128
// (eight 16-token pages). The two query tiles share every K / V tile and alternate on the tensor core, so the softmax of
// one runs while the MMAs of the other execute.
//   warp 0      : TMA producer - both Q tiles once, then per key tile sixteen boxes for K and sixteen for V (a page is
//                 [16 keys x 64 values] per half of the head dimension, 128-byte swizzled); K and V have their own
//                 two-deep rings, because a K tile is free a whole step before its V tile
//   warp 1      : MMA issuer (one thread) - S_w = Q_w K_j^T into tile w's score columns, O_w += P_w V_j with P_w read
//                 from tensor memory (the A operand) and V as it lies in the cache ([key][value], MN-major B operand)
//   warps 2..5  : softmax of tile a, warps 6..9 of tile b, one query row per thread (TMEM lane = row): the whole score
//                 row comes into registers with one wait, P = exp2(S * scale - m) goes back as packed bf16 over the
//                 first 64 score columns. The output accumulator stays in tensor memory; it is rescaled only when a
//                 row's maximum has grown by more than 2^8 since the scale in use was chosen (the probabilities are
//                 then at most 256, exact enough in bf16, and the final division by the row sum takes the scale out).
// TMEM columns: S_a [0,128) | S_b [128,256) | O_a [256,384) | O_b [384,512).
// Causal masking by position (queries are the last q_len positions of their sequence, so chunked prefill and cached
// prefixes work); key tiles beyond a query tile's last position are never loaded. CTAs with the most key tiles are
// scheduled first.
//
// Key and value widths up to 128 (multiples of 8, not necessarily equal: a 64-wide half that reaches beyond the stored
// width is filled with zeros by the TMA), optional sliding window or chunks of positions (key tiles before what a tile's
// rows can see are skipped) and sink logits. Same
// online-softmax recurrence and semantics as attn_prefill_kernel in attention.cu and as the reference's blockwise attention (eredu/src/backend/mlx/nn/attention.rs:346-436,
// runtime/cache/kv.rs:2267-2436). Every wait is bounded; on expiry the status word is set and the CTA leaves through the
// common exit (TMEM is freed there).
#include <cuda_bf16.h>

#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/launch_count.h"
#include "../common/pooled.cuh"
#include "../common/ptx.cuh"
#include "../common/tma_host.h"
#include "../common/trace.cuh"

namespace eredu {

struct AttnTcParams {
  __nv_bfloat16* out;          // [tokens, n_q, dv]
  const int* block_table;      // [batch, max_pages]
  const int* seq_lens;         // kv length after this call, per sequence
  const int* cu_q;             // [batch + 1] query-row offsets
  const float* sinks;          // optional [n_q_heads]: logit of a virtual key with zero value (enters the normaliser only)
  int max_pages;
  int n_q_heads, n_kv_heads;
  int window;                  // 0: none; else a query at position p sees keys in (p - window, p]
  int chunk;                   // > 0 (window 0): a query sees the keys of its own chunk of positions
  int dk, dv;                  // key / value width of a head (multiples of 8); the rest of a 64-wide half reads as zero
  float scale_log2;
  int* status;
  // ROWS form: table {first query row, queries, first context row, context rows} per sequence instead of the four arrays above; keys
  // of dk = dim + rot, of which the last rot are the shared part
  const int4* table;
  const __nv_bfloat16* gate;   // optional [tokens, ldg]: column head * dv + i
  long long ldg;
  int rot;
  // POOL form (window > 0): all whole blocks of `pool` tokens of a sequence as dense rows from pool_first[b] on
  const int* pool_first;
  int pool;
};

constexpr int kTcThreads = 320;
constexpr int kTcTile = 128;            // query rows per tile and keys per tile
constexpr int kTcRows = 2 * kTcTile;    // query rows per CTA
constexpr int kTcHalf = 128 * 64 * 2;   // one [128 rows][64 bf16] swizzled half tile: 16 KB
// shared memory: Q_a, Q_b (NK halves each) | K ring (2 x NK halves) | V ring (2 x NV halves) | barriers
// Three key halves and two value halves leave room for one V stage only.
constexpr int tc_v_stages(int nk, int nv) { return nk + nv > 4 ? 1 : 2; }
constexpr int tc_smem(int nk, int nv) { return 1024 + (4 * nk + tc_v_stages(nk, nv) * nv) * kTcHalf + 256; }
// A quarter of the exponentials as a polynomial on the FMA pipe (build option). Measured slower here (1153 against 1192
// TFLOP/s at 32k tokens, 1112 against 1170 at 8k): the softmax warps are bound by instruction issue, not by the
// special-function unit, so the extra FMA-pipe instructions cost more than the unit they relieve.
#ifndef EREDU_ATTN_POLY_EXP
#define EREDU_ATTN_POLY_EXP 0
#endif
constexpr bool kTcPolyExp = EREDU_ATTN_POLY_EXP != 0;
constexpr float kTcRescale = 8.f;       // log2 units a row maximum may outgrow the scale in use

// MN-major operand tile stored as [k rows][64 bf16] (128-byte rows, 128B swizzle): 64-element blocks along MN are `lbo`
// bytes apart, 8-row groups along K are 1024 bytes apart. Advancing K by 16 = +2048 bytes on the start address.
__device__ __forceinline__ uint64_t umma_desc_mn_sw128(uint32_t smem_addr, uint32_t lbo_bytes) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((smem_addr & 0x3FFFF) >> 4);
  d |= static_cast<uint64_t>(lbo_bytes >> 4) << 16;
  d |= static_cast<uint64_t>(1024 >> 4) << 32;
  d |= static_cast<uint64_t>(1) << 46;
  d |= static_cast<uint64_t>(2) << 61;
  return d;
}
constexpr uint32_t kIdescQK = umma_idesc_bf16(128, 128);                 // both operands K-major

__device__ __forceinline__ void tma_load_4d(void* smem_dst, const CUtensorMap* map, int x, int y, int z, int w, uint64_t* bar) {
  asm volatile(
      "cp.async.bulk.tensor.4d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4, %5}], [%6];"
      :
      : "r"(smem_u32(smem_dst)), "l"(reinterpret_cast<uint64_t>(map)), "r"(x), "r"(y), "r"(z), "r"(w), "r"(smem_u32(bar))
      : "memory");
}

// First key position a query at `pos` can see.
__device__ __forceinline__ int tc_lowest_key(const AttnTcParams& p, int pos) {
  if (p.window > 0) return max(0, pos - p.window + 1);
  return p.chunk > 0 ? pos - pos % p.chunk : 0;
}

// Order in which query tiles are taken, longest first: the last positions of a causal prompt, the last tiles of every chunk.
__device__ __forceinline__ int tc_query_tile(const AttnTcParams& p, int tiles, int y) {
  const int per = p.chunk / kTcRows;                                    // query tiles of a chunk
  if (per < 2) return tiles - 1 - y;
  for (int r = min(per, tiles) - 1; r > 0; --r) {
    const int n = (tiles - r + per - 1) / per;
    if (y < n) return r + y * per;
    y -= n;
  }
  return y * per;
}

// NK / NV: 64-wide halves of the key and of the value width. POOL: key tiles of 128 mean keys come in front of the tiles of the window; tile
// index u walks the pooled tiles 0 .. pooled - 1, then the token tiles from j0 on.
template <int NK, int NV, bool ROWS, bool POOL>
__global__ void __launch_bounds__(kTcThreads, 1)
attn_prefill_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                       const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmR,
                       const __grid_constant__ CUtensorMap tmS, const AttnTcParams p) {
  constexpr int VST = tc_v_stages(NK, NV);
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const uint32_t kIdescPV = umma_idesc_bf16(128, (p.dv + 15) & ~15) | (1u << 16);  // B (= V) MN-major, N = value width
  const int k_steps = (p.dk + 15) >> 4, o_steps = (p.dv + 15) >> 4;
  uint8_t* q_s = smem;                                                 // tile w at + w * NK halves
  uint8_t* k_s = q_s + 2 * NK * kTcHalf;                               // stage s at + s * NK (K), s * NV (V) halves
  uint8_t* v_s = k_s + 2 * NK * kTcHalf;
  uint64_t* bars = reinterpret_cast<uint64_t*>(v_s + VST * NV * kTcHalf);
  uint64_t* q_full = bars;                  // 1
  uint64_t* k_full = bars + 1;              // [2]
  uint64_t* k_empty = bars + 3;             // [2]
  uint64_t* v_full = bars + 5;              // [2]
  uint64_t* v_empty = bars + 7;             // [2]
  uint64_t* s_full = bars + 9;              // [2] per query tile
  uint64_t* p_full = bars + 11;             // [2] per query tile, 128 arrivals
  uint64_t* o_final = bars + 13;            // [2] per query tile
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 16);

  pdl_launch_early();
  trace_mark(kTraceAttnPrefill, kTraceStart);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // heads vary fastest: the first wave holds the longest query tiles of every head (longest-first balances the causal
  // triangle), and neighbouring CTAs are query heads of one key / value head reading the same pages
  const int b = blockIdx.z, head = blockIdx.x, qt = tc_query_tile(p, gridDim.y, blockIdx.y);
  const int4 seq = ROWS ? p.table[b] : make_int4(p.cu_q[b], p.cu_q[b + 1] - p.cu_q[b], 0, p.seq_lens[b]);
  const int q0 = seq.x, q_len = seq.y, kv_len = seq.w;
  const int row0 = qt * kTcRows;
  if (row0 >= q_len) return;                                            // uniform: before any barrier or allocation
  const int kv_head = head / (p.n_q_heads / p.n_kv_heads);
  const int pos0 = kv_len - q_len + row0;                               // position of the CTA's first query row
  // causal: nothing beyond the position of a tile's last row
  const int n_a = min(kv_len - 1, pos0 + kTcTile - 1) / kTcTile + 1;
  const int n_b = row0 + kTcTile < q_len ? min(kv_len - 1, pos0 + kTcRows - 1) / kTcTile + 1 : 0;
  const int n_tiles = max(n_a, n_b);
  // window / chunk: key tiles that lie wholly before what a tile's FIRST row sees are skipped
  const int j0_a = tc_lowest_key(p, pos0) / kTcTile;
  const int j0_b = tc_lowest_key(p, pos0 + kTcTile) / kTcTile;
  const int j0 = n_b > 0 ? min(j0_a, j0_b) : j0_a;
  // pooled tiles some row of query tile a, b sees (the last row sees most)
  const int np_a = POOL ? (pooled_seen(min(kv_len - 1, pos0 + kTcTile - 1), p.window, p.pool) + kTcTile - 1) / kTcTile : 0;
  const int np_b = POOL && n_b > 0 ? (pooled_seen(min(kv_len - 1, pos0 + kTcRows - 1), p.window, p.pool) + kTcTile - 1) / kTcTile : 0;
  const int pooled = max(np_a, np_b);
  const int total = pooled + n_tiles - j0;                              // tiles this CTA walks

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(&k_full[s], 1);
      mbar_init(&k_empty[s], 1);
      mbar_init(&v_full[s], 1);
      mbar_init(&v_empty[s], 1);
      mbar_init(&s_full[s], 1);
      mbar_init(&p_full[s], 128);
      mbar_init(&o_final[s], 1);
    }
    fence_mbar_init();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
    if (ROWS || POOL) tma_prefetch_desc(&tmR);
    if (POOL) tma_prefetch_desc(&tmS);
  }
  if (warp == 0) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = *tmem_slot;
  pdl_wait();
  trace_mark(kTraceAttnPrefill, kTraceAfterWait);
  pdl_launch_dependents();

  bool ok = true;
  if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer
    if (lane == 0) {
      mbar_arrive_expect_tx(q_full, 2 * NK * kTcHalf);
      for (int w = 0; w < 2; ++w)
        for (int h = 0; h < NK; ++h)
          // ROWS: the last half starts where the shared part does; a box that reaches beyond the per-head part meets zeros on the key side
          tma_load_3d(q_s + (w * NK + h) * kTcHalf, &tmQ, ROWS && h == NK - 1 ? p.dk - p.rot : h * 64, head, q0 + row0 + w * kTcTile, q_full);
      const int* pages = p.block_table + static_cast<size_t>(b) * p.max_pages;
      const int pool_row = POOL ? p.pool_first[b] : 0;
      for (int jj = 0; jj < total && ok; ++jj) {
        const bool means = POOL && jj < pooled;
        const int j = means ? jj : j0 + jj - pooled;                     // key tile; jj counts this CTA's iterations
        const int s = jj & 1;
        const uint32_t reuse_parity = ((jj >> 1) - 1) & 1;
        const int sv = VST == 2 ? s : 0;
        int page[8];
        if (!ROWS && !means) {
#pragma unroll
          for (int pg = 0; pg < 8; ++pg) {
            const int page_index = j * 8 + pg;
            page[pg] = page_index < p.max_pages ? pages[page_index] : 0;            // beyond the table: the reserved page (masked)
          }
        }
        if (jj >= 2) ok = mbar_wait(&k_empty[s], reuse_parity, p.status, kStatusSmemEmptyTimeout);
        if (!ok) break;
        mbar_arrive_expect_tx(&k_full[s], NK * kTcHalf);
        if (ROWS) {
          for (int h = 0; h + 1 < NK; ++h) tma_load_3d(k_s + (s * NK + h) * kTcHalf, &tmK, h * 64, head, seq.z + j * kTcTile, &k_full[s]);
          tma_load_2d(k_s + (s * NK + NK - 1) * kTcHalf, &tmR, 0, seq.z + j * kTcTile, &k_full[s]);
        }
        if (means) {
          for (int h = 0; h < NK; ++h) tma_load_3d(k_s + (s * NK + h) * kTcHalf, &tmR, h * 64, kv_head, pool_row + j * kTcTile, &k_full[s]);
        } else {
#pragma unroll
          for (int pg = 0; pg < (ROWS ? 0 : 8); ++pg)
            for (int h = 0; h < NK; ++h) tma_load_4d(k_s + (s * NK + h) * kTcHalf + pg * 2048, &tmK, h * 64, 0, kv_head, page[pg], &k_full[s]);
        }
        if (jj >= VST) ok = mbar_wait(&v_empty[sv], VST == 2 ? reuse_parity : (jj - 1) & 1, p.status, kStatusSmemEmptyTimeout);
        if (!ok) break;
        mbar_arrive_expect_tx(&v_full[sv], NV * kTcHalf);
        if (ROWS)
          for (int h = 0; h < NV; ++h) tma_load_3d(v_s + (sv * NV + h) * kTcHalf, &tmV, h * 64, head, seq.z + j * kTcTile, &v_full[sv]);
        if (means) {
          for (int h = 0; h < NV; ++h) tma_load_3d(v_s + (sv * NV + h) * kTcHalf, &tmS, h * 64, kv_head, pool_row + j * kTcTile, &v_full[sv]);
        } else {
#pragma unroll
          for (int pg = 0; pg < (ROWS ? 0 : 8); ++pg)
            for (int h = 0; h < NV; ++h) tma_load_4d(v_s + (sv * NV + h) * kTcHalf + pg * 2048, &tmV, h * 64, 0, kv_head, page[pg], &v_full[sv]);
        }
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    if (lane == 0) {
      const uint32_t q_addr = smem_u32(q_s);
      // jj: this CTA's iteration (selects the K / V stage); tile w is active on key tiles [first_w, n_w)
      const int first[2] = {j0_a, j0_b}, last[2] = {n_a, n_b};
      auto issue_s = [&](int w, int jj) {
        const uint32_t qa = q_addr + w * NK * kTcHalf;
        const uint32_t ka = smem_u32(k_s + (jj & 1) * NK * kTcHalf);
        const uint32_t d = tmem + w * 128;
#pragma unroll
        for (int kk = 0; kk < NK * 4; ++kk) {      // K = key width: four 16-steps per 64-wide half
          if (ROWS ? (kk & 3) * 16 >= (kk >> 2 == NK - 1 ? p.rot : p.dk - p.rot - (kk >> 2) * 64) : kk >= k_steps) continue;
          const uint32_t off = (kk >> 2) * kTcHalf + (kk & 3) * 32;
          umma_f16(d, umma_desc_k_sw128(qa + off), umma_desc_k_sw128(ka + off), kIdescQK, kk > 0 ? 1u : 0u);
        }
        umma_commit(&s_full[w]);
      };
      auto issue_pv = [&](int w, int jj, bool fresh) {
        const uint32_t va = smem_u32(v_s + (VST == 2 ? jj & 1 : 0) * NV * kTcHalf);
#pragma unroll
        for (int kk = 0; kk < 8; ++kk)             // K = keys: P from tensor memory (8 columns per step), V MN-major (2048 bytes per step)
          umma_f16_ts(tmem + 256 + w * 128, tmem + w * 128 + kk * 8, umma_desc_mn_sw128(va + kk * 2048, kTcHalf), kIdescPV,
                      (!fresh || kk > 0) ? 1u : 0u);
      };
      const int seen[2] = {np_a, np_b};
      // u counts this CTA's iterations; a query tile's last one is a token tile
      auto active = [&](int w, int u) { return POOL && u < pooled ? u < seen[w] : u >= pooled + first[w] - j0 && u < pooled + last[w] - j0; };
      ok = mbar_wait(q_full, 0, p.status, kStatusTmaFullTimeout);
      if (ok) ok = mbar_wait(&k_full[0], 0, p.status, kStatusTmaFullTimeout);
      if (ok) {
        tc_fence_after_sync();
        if (active(0, 0)) issue_s(0, 0);
        if (active(1, 0)) issue_s(1, 0);
        umma_commit(&k_empty[0]);
      }
      int done[2] = {0, 0};                        // softmax rounds completed per tile: parity of p_full
      for (int jj = 0; jj < total && ok; ++jj) {
        const bool next = jj + 1 < total;
        bool k_ready = false;
        ok = mbar_wait(&v_full[VST == 2 ? jj & 1 : 0], (VST == 2 ? jj >> 1 : jj) & 1, p.status, kStatusTmaFullTimeout);
        for (int w = 0; w < 2 && ok; ++w) {
          if (active(w, jj)) {
            ok = mbar_wait(&p_full[w], done[w] & 1, p.status, kStatusAccumTimeout);   // P_w(j) is in tensor memory, O_w is rescaled
            if (!ok) break;
            tc_fence_after_sync();
            issue_pv(w, jj, done[w] == 0);
            ++done[w];
          }
          if (w == 1) umma_commit(&v_empty[VST == 2 ? jj & 1 : 0]);
          if (active(w, jj + 1)) {
            if (!k_ready) {
              ok = mbar_wait(&k_full[(jj + 1) & 1], ((jj + 1) >> 1) & 1, p.status, kStatusTmaFullTimeout);
              if (!ok) break;
              tc_fence_after_sync();
              k_ready = true;
            }
            issue_s(w, jj + 1);
          } else if (jj + 1 == pooled + last[w] - j0) {
            umma_commit(&o_final[w]);
          }
        }
        if (ok && next) umma_commit(&k_empty[(jj + 1) & 1]);
      }
    }
  } else {
    // ------------------------------------------------------------------ softmax, one row per thread
    const int w = (warp - 2) >> 2;                                       // query tile of this warp
    const int n_w = w == 0 ? n_a : n_b;
    const int j0_w = w == 0 ? j0_a : j0_b;
    const int quarter = warp & 3;                                        // TMEM lanes this warp may touch
    const int row = quarter * 32 + lane;
    const int tile_row0 = row0 + w * kTcTile;
    const int tile_pos0 = pos0 + w * kTcTile;
    const int qpos = tile_pos0 + row;
    const uint32_t lane_addr = static_cast<uint32_t>(quarter * 32) << 16;
    const uint32_t s_addr = tmem + lane_addr + w * 128;
    const uint32_t o_addr = tmem + lane_addr + 256 + w * 128;
    float m = -INFINITY, l = 0.f;                                        // -inf: this row has not seen a key yet
    const int np_w = w == 0 ? np_a : np_b;
    for (int it = 0; it < np_w + n_w - j0_w && ok; ++it) {               // this tile's round: parity of its barriers
      const bool means = POOL && it < np_w;
      const int j = means ? it : j0_w + it - np_w;
      ok = mbar_wait(&s_full[w], it & 1, p.status, kStatusAccumTimeout);
      if (!ok) break;
      tc_fence_after_sync();
      uint32_t sc[8][16];
#pragma unroll
      for (int c = 0; c < 8; ++c) tmem_ld16(s_addr + c * 16, sc[c]);
      tmem_wait_ld();
      const int key0 = j * kTcTile;
      const bool before = key0 < tc_lowest_key(p, tile_pos0 + kTcTile - 1);     // some row's visible keys start inside or after this tile
      if (means) {
        const int blocks = pooled_seen(qpos, p.window, p.pool) - key0;   // of this tile's
        if (key0 + kTcTile > pooled_seen(tile_pos0, p.window, p.pool)) {
#pragma unroll
          for (int c = 0; c < 8; ++c)
#pragma unroll
            for (int i = 0; i < 16; ++i)
              if (c * 16 + i >= blocks) sc[c][i] = 0xFF800000u;
        }
      } else if (key0 + kTcTile - 1 > tile_pos0 || key0 + kTcTile > kv_len || before) {   // some (row, key) of the tile is masked: -inf gives p = 0
        const int visible = min(qpos, kv_len - 1) - key0;                // keys hidden .. visible of this tile are seen by this row
        const int hidden = tc_lowest_key(p, qpos) - key0;
#pragma unroll
        for (int c = 0; c < 8; ++c)
#pragma unroll
          for (int i = 0; i < 16; ++i)
            if (c * 16 + i > visible || c * 16 + i < hidden) sc[c][i] = 0xFF800000u;
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};      // four chains of three-input maxima
#pragma unroll
      for (int c = 0; c < 8; ++c)
#pragma unroll
        for (int i = 0; i < 16; i += 2) mx4[(i >> 1) & 3] = max3(mx4[(i >> 1) & 3], __uint_as_float(sc[c][i]), __uint_as_float(sc[c][i + 1]));
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      const float m_new = mx * p.scale_log2;                             // -inf for a fully masked row: every comparison below is false
      bool grow = false;
      if (m == -INFINITY) {
        m = m_new;                                                       // what the row added so far is zero
      } else {
        grow = m_new > m + kTcRescale;
      }
      if (it > 0) {
        if (__any_sync(0xffffffffu, grow)) {                             // O_w(j - 1) is complete: s_full followed it on the tensor core
          const float alpha = grow ? ex2_approx(m - m_new) : 1.f;
          if (grow) m = m_new;
          l *= alpha;
#pragma unroll 1
          for (int c = 0; c < o_steps; ++c) {
            uint32_t r[16];
            tmem_ld16(o_addr + c * 16, r);
            tmem_wait_ld();
#pragma unroll
            for (int i = 0; i < 16; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * alpha);
            tmem_st16(o_addr + c * 16, r);
          }
        }
      }
      // p = exp2(s * scale - m), two values per FMA / add; sums in four chains
      const float shift = m == -INFINITY ? 0.f : -m;
      const uint64_t scale2 = pack_f32x2(p.scale_log2, p.scale_log2), shift2 = pack_f32x2(shift, shift);
      uint64_t acc[4] = {0ull, 0ull, 0ull, 0ull};
#pragma unroll
      for (int c2 = 0; c2 < 4; ++c2) {
        uint32_t packed[16];
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          const int c = c2 * 2 + (i >> 4), e = i & 15;
          float t0, t1;
          unpack_f32x2(fma_f32x2(pack_b32x2(sc[c][e], sc[c][e + 1]), scale2, shift2), t0, t1);
          // every fourth pair takes the polynomial on the FMA pipe instead of the special-function unit
          const bool poly = kTcPolyExp && ((i >> 1) & 3) == 3;
          const float p0 = poly ? ex2_poly(t0) : ex2_approx(t0), p1 = poly ? ex2_poly(t1) : ex2_approx(t1);
          acc[(i >> 1) & 3] = add_f32x2(acc[(i >> 1) & 3], pack_f32x2(p0, p1));
          packed[i >> 1] = pack_bf16x2(p0, p1);
        }
        tmem_st16(s_addr + c2 * 16, packed);
      }
      tmem_wait_st();
      tc_fence_before_sync();
      mbar_arrive(&p_full[w]);
      float s0, s1;
      unpack_f32x2(add_f32x2(add_f32x2(acc[0], acc[1]), add_f32x2(acc[2], acc[3])), s0, s1);
      l += s0 + s1;
    }
    if (ok && n_w > 0) ok = mbar_wait(&o_final[w], 0, p.status, kStatusAccumTimeout);
    if (ok && n_w > 0) {
      tc_fence_after_sync();
      const bool store = tile_row0 + row < q_len;
      if (p.sinks != nullptr) l += ex2_approx(p.sinks[head] * 1.4426950408889634f - m);
      const float inv = l > 0.f ? 1.f / l : 0.f;
      uint4* dst = reinterpret_cast<uint4*>(p.out + (static_cast<size_t>(q0 + tile_row0 + row) * p.n_q_heads + head) * p.dv);
#pragma unroll 1
      for (int c = 0; c < o_steps; ++c) {
        uint32_t r[16];
        tmem_ld16(o_addr + c * 16, r);
        tmem_wait_ld();
        if (store) {
          if (ROWS && p.gate != nullptr) {
            const uint4* gp = reinterpret_cast<const uint4*>(p.gate + static_cast<size_t>(q0 + tile_row0 + row) * p.ldg + head * p.dv + c * 16);
            const uint4 g0 = gp[0], g1 = c * 16 + 8 < p.dv ? gp[1] : make_uint4(0u, 0u, 0u, 0u);
            const uint32_t gw[8] = {g0.x, g0.y, g0.z, g0.w, g1.x, g1.y, g1.z, g1.w};
#pragma unroll
            for (int i = 0; i < 8; ++i) {
              r[2 * i] = __float_as_uint(__uint_as_float(r[2 * i]) * sigmoid_fast(bf16_lo(gw[i])));
              r[2 * i + 1] = __float_as_uint(__uint_as_float(r[2 * i + 1]) * sigmoid_fast(bf16_hi(gw[i])));
            }
          }
          uint4 v0, v1;
          v0.x = pack_bf16x2(__uint_as_float(r[0]) * inv, __uint_as_float(r[1]) * inv);
          v0.y = pack_bf16x2(__uint_as_float(r[2]) * inv, __uint_as_float(r[3]) * inv);
          v0.z = pack_bf16x2(__uint_as_float(r[4]) * inv, __uint_as_float(r[5]) * inv);
          v0.w = pack_bf16x2(__uint_as_float(r[6]) * inv, __uint_as_float(r[7]) * inv);
          v1.x = pack_bf16x2(__uint_as_float(r[8]) * inv, __uint_as_float(r[9]) * inv);
          v1.y = pack_bf16x2(__uint_as_float(r[10]) * inv, __uint_as_float(r[11]) * inv);
          v1.z = pack_bf16x2(__uint_as_float(r[12]) * inv, __uint_as_float(r[13]) * inv);
          v1.w = pack_bf16x2(__uint_as_float(r[14]) * inv, __uint_as_float(r[15]) * inv);
          dst[c * 2] = v0;
          if (c * 16 + 8 < p.dv) dst[c * 2 + 1] = v1;
        }
      }
    }
  }
  // common exit: every role comes here, also after a timed-out wait; the tensor memory goes back
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 0) tmem_dealloc(tmem, 512);
  trace_mark(kTraceAttnPrefill, kTraceEnd);
}

}  // namespace eredu

using namespace eredu;

// Causal prefill attention over the paged cache, key / value widths up to 128, optional window or chunks and sink logits.
// q: [tokens, n_q, key_dim] bf16 (contiguous); k_cache / v_cache: [pages, n_kv, 16, width] bf16 (contiguous); sinks: fp32 [n_q] or
// null. Same arguments as eredu_attn_prefill otherwise. Returns -2 for shapes it does not take.
template <int NK, int NV, bool ROWS = false, bool POOL = false>
static int launch_attn_tc(const CUtensorMap& tmQ, const CUtensorMap& tmK, const CUtensorMap& tmV, const CUtensorMap& tmR, const CUtensorMap& tmS,
                          const AttnTcParams& p, dim3 grid, cudaStream_t stream) {
  static bool configured[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !configured[dev]) {
    if (cudaFuncSetAttribute(attn_prefill_tc_kernel<NK, NV, ROWS, POOL>, cudaFuncAttributeMaxDynamicSharedMemorySize, tc_smem(NK, NV)) != cudaSuccess) return -1;
    configured[dev] = true;
  }
  return static_cast<int>(launch_pdl(attn_prefill_tc_kernel<NK, NV, ROWS, POOL>, grid, dim3(kTcThreads), tc_smem(NK, NV), stream, tmQ, tmK, tmV, tmR, tmS, p));
}

static int attn_prefill_tc_impl(const void* q, const void* k_cache, const void* v_cache, const void* k_rows, const void* v_rows, void* out,
                                const int* block_table, const int* seq_lens, const int* cu_q, const int* pool_first, const float* sinks, int batch,
                                int total_q, int max_q_len, int max_pages, int num_pages, int rows, int n_q_heads, int n_kv_heads, int key_dim,
                                int value_dim, int window, int chunk, int pool, float scale, int* status, cudaStream_t stream) {
  if (key_dim <= 0 || key_dim > 128 || key_dim % 8 != 0 || value_dim <= 0 || value_dim > 128 || value_dim % 8 != 0 || batch <= 0 ||
      total_q <= 0 || n_kv_heads <= 0 || n_q_heads % n_kv_heads != 0 || window < 0 || chunk < 0)
    return -2;
  const uint64_t D = static_cast<uint64_t>(key_dim), V = static_cast<uint64_t>(value_dim);
  CUtensorMap tmQ, tmK, tmV;
  // q as [tokens][heads][D]: box = 128 tokens x 1 head x 64 values
  int r = make_tma_3d(&tmQ, q, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, D, static_cast<uint64_t>(n_q_heads),
                      static_cast<uint64_t>(total_q), D * 2, static_cast<uint64_t>(n_q_heads) * D * 2, 64, 1, 128);
  if (r != 0) return -100 + r;
  r = make_tma_4d(&tmK, k_cache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, D, 16, static_cast<uint64_t>(n_kv_heads),
                  static_cast<uint64_t>(num_pages), D * 2, 16 * D * 2, static_cast<uint64_t>(n_kv_heads) * 16 * D * 2, 64, 16, 1, 1);
  if (r != 0) return -200 + r;
  r = make_tma_4d(&tmV, v_cache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, V, 16, static_cast<uint64_t>(n_kv_heads),
                  static_cast<uint64_t>(num_pages), V * 2, 16 * V * 2, static_cast<uint64_t>(n_kv_heads) * 16 * V * 2, 64, 16, 1, 1);
  if (r != 0) return -300 + r;
  AttnTcParams p = {};
  p.out = static_cast<__nv_bfloat16*>(out);
  p.block_table = block_table;
  p.seq_lens = seq_lens;
  p.cu_q = cu_q;
  p.sinks = sinks;
  p.max_pages = max_pages;
  p.n_q_heads = n_q_heads;
  p.n_kv_heads = n_kv_heads;
  p.window = window;
  p.chunk = chunk;
  p.dk = key_dim;
  p.dv = value_dim;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.status = status;
  dim3 grid(n_q_heads, (max_q_len + kTcRows - 1) / kTcRows, batch);
  int e;
  if (pool > 0) {
    // no whole block anywhere yet: the maps of the caches stand in, and no tile of means is walked
    CUtensorMap tmR = tmK, tmS = tmV;
    const uint64_t G = static_cast<uint64_t>(n_kv_heads), n = static_cast<uint64_t>(rows);
    if (rows > 0) {
      r = make_tma_3d(&tmR, k_rows, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, D, G, n, D * 2, G * D * 2, 64, 1, 128);
      if (r != 0) return -400 + r;
      r = make_tma_3d(&tmS, v_rows, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, V, G, n, V * 2, G * V * 2, 64, 1, 128);
      if (r != 0) return -500 + r;
    }
    p.pool = pool;
    p.pool_first = pool_first;
#define ER_POOLED(NK_, NV_) e = launch_attn_tc<NK_, NV_, false, true>(tmQ, tmK, tmV, tmR, tmS, p, grid, stream)
    if (key_dim > 64 && value_dim > 64) ER_POOLED(2, 2);
    else if (key_dim > 64) ER_POOLED(2, 1);
    else if (value_dim > 64) ER_POOLED(1, 2);
    else ER_POOLED(1, 1);
#undef ER_POOLED
    eredu_count_launches(1);
    return e;
  }
  if (key_dim > 64) e = value_dim > 64 ? launch_attn_tc<2, 2>(tmQ, tmK, tmV, tmK, tmV, p, grid, stream) : launch_attn_tc<2, 1>(tmQ, tmK, tmV, tmK, tmV, p, grid, stream);
  else e = value_dim > 64 ? launch_attn_tc<1, 2>(tmQ, tmK, tmV, tmK, tmV, p, grid, stream) : launch_attn_tc<1, 1>(tmQ, tmK, tmV, tmK, tmV, p, grid, stream);
  eredu_count_launches(1);
  return e;
}

extern "C" int eredu_attn_prefill_tc(const void* q, const void* k_cache, const void* v_cache, void* out, const int* block_table,
                                     const int* seq_lens, const int* cu_q, const float* sinks, int batch, int total_q, int max_q_len,
                                     int max_pages, int num_pages, int n_q_heads, int n_kv_heads, int key_dim, int value_dim, int window,
                                     int chunk, float scale, int* status, cudaStream_t stream) {
  return attn_prefill_tc_impl(q, k_cache, v_cache, nullptr, nullptr, out, block_table, seq_lens, cu_q, nullptr, sinks, batch, total_q, max_q_len,
                              max_pages, num_pages, 0, n_q_heads, n_kv_heads, key_dim, value_dim, window, chunk, 0, scale, status, stream);
}

// The POOL form: over the `window` newest tokens and the means of the blocks of `pool` tokens that end before them. k_rows / v_rows [rows,
// n_kv, width] bf16: all whole blocks of sequence b from row pool_first[b] on (null when rows = 0: no sequence has one).
extern "C" int eredu_attn_prefill_tc_pooled(const void* q, const void* k_cache, const void* v_cache, const void* k_rows, const void* v_rows, void* out,
                                            const int* block_table, const int* seq_lens, const int* cu_q, const int* pool_first, int batch,
                                            int total_q, int max_q_len, int max_pages, int num_pages, int rows, int n_q_heads, int n_kv_heads,
                                            int key_dim, int value_dim, int window, int pool, float scale, int* status, cudaStream_t stream) {
  if (window <= 0 || pool <= 0 || rows < 0 || pool_first == nullptr || (rows > 0 && (k_rows == nullptr || v_rows == nullptr))) return -2;
  return attn_prefill_tc_impl(q, k_cache, v_cache, k_rows, v_rows, out, block_table, seq_lens, cu_q, pool_first, nullptr, batch, total_q, max_q_len,
                              max_pages, num_pages, rows, n_q_heads, n_kv_heads, key_dim, value_dim, window, 0, pool, scale, status, stream);
}

// The ROWS form. q [total_q rows of ldq elements], head h at column h * (dim + rot): [per-head part (dim) | shared part (rot)]; k [rows of
// ldkv], head h at h * dim; v [rows of ldkv], head h at h * value_dim; kr [rows of ldkr]: the shared key part; table [n_seq] int4
// {first query row, queries, first context row, context rows}: the queries are the last positions of their context rows. gate
// [total_q rows of ldg] or null, column h * value_dim + i. out [total_q, heads, value_dim]. dim, value_dim <= 128, rot <= 64, all
// multiples of 8, pitches and pointers 16-byte aligned.
extern "C" int eredu_attn_prefill_rows(const void* q, const void* k, const void* v, const void* kr, const void* gate, const float* sinks,
                                       void* out, const int* table, int n_seq, int total_q, int rows, int max_q, int heads, int dim,
                                       int rot, int value_dim, int window, long long ldq, long long ldkv, long long ldkr, long long ldg,
                                       float scale, int* status, cudaStream_t stream) {
  if (n_seq <= 0 || max_q <= 0 || rows <= 0) return 0;
  if (dim <= 0 || dim > 128 || dim % 8 != 0 || rot <= 0 || rot > 64 || rot % 8 != 0 || value_dim <= 0 || value_dim > 128 ||
      value_dim % 8 != 0 || heads <= 0 || window < 0 || n_seq > 65535)
    return -2;
  const uint64_t D = static_cast<uint64_t>(dim), R = static_cast<uint64_t>(rot), V = static_cast<uint64_t>(value_dim);
  const uint64_t H = static_cast<uint64_t>(heads);
  CUtensorMap tmQ, tmK, tmV, tmR;
  int r = make_tma_3d(&tmQ, q, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, D + R, H, static_cast<uint64_t>(total_q), (D + R) * 2, ldq * 2, 64, 1, 128);
  if (r != 0) return -100 + r;
  r = make_tma_3d(&tmK, k, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, D, H, static_cast<uint64_t>(rows), D * 2, ldkv * 2, 64, 1, 128);
  if (r != 0) return -200 + r;
  r = make_tma_3d(&tmV, v, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, V, H, static_cast<uint64_t>(rows), V * 2, ldkv * 2, 64, 1, 128);
  if (r != 0) return -300 + r;
  r = make_tma_2d(&tmR, kr, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, static_cast<uint64_t>(rows), R, static_cast<uint64_t>(ldkr), 128, 64);
  if (r != 0) return -400 + r;
  AttnTcParams p = {};
  p.out = static_cast<__nv_bfloat16*>(out);
  p.sinks = sinks;
  p.n_q_heads = heads;
  p.n_kv_heads = heads;
  p.window = window;
  p.dk = dim + rot;
  p.dv = value_dim;
  p.rot = rot;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.status = status;
  p.table = reinterpret_cast<const int4*>(table);
  p.gate = static_cast<const __nv_bfloat16*>(gate);
  p.ldg = ldg;
  const dim3 grid(heads, (max_q + kTcRows - 1) / kTcRows, n_seq);
  if (grid.y > 65535) return -2;
  int e;
#define ER_ROWS(NK_) \
  e = value_dim > 64 ? launch_attn_tc<NK_, 2, true>(tmQ, tmK, tmV, tmR, tmV, p, grid, stream) : launch_attn_tc<NK_, 1, true>(tmQ, tmK, tmV, tmR, tmV, p, grid, stream)
  if (dim > 64) ER_ROWS(3);
  else ER_ROWS(2);
#undef ER_ROWS
  eredu_count_launches(1);
  return e;
}
