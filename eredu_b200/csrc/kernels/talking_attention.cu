// Paged attention whose heads exchange their scores before the softmax: the score of head h is sum_g talk[h, g] cap(scale q_g . k_g),
// cap(s) = softcap tanh(s / softcap), over a sliding window and the first tokens of the sequence, with a sink per head.
//
// A query's heads cannot be computed apart, so a group of warps owns ALL heads of a few queries and walks the visible pages of 16 keys:
//   score    S^T[key, column] = K Q^T per key / value head on the tensor cores, a column being one (query, head of the group); the cap in
//            fp32; S goes to shared memory with the heads of a (query, key) pair side by side
//   mix      S'[head, pair] = talk S on the tensor cores: S as three bf16 pieces (exact), talk is bf16 itself, fp32 accumulation
//   combine  online softmax per column and O^T[value dim, column] += V^T P^T, O in registers
// The score step of page i + 1 and the combine step of page i lie between the same two barriers; keys and values arrive by cp.async two
// stages deep. Prompts: one group of up to 16 warps and as many queries as fit its registers. Decode steps: several groups per CTA, each
// with pages of its own, and the CTAs of a cluster share a sequence's keys; partial results meet in (distributed) shared memory.
//
// Prompts of the usual head sizes have kernels of their own. They use that exponents of fp32 and bf16 reach far: the mix step forms exp(S')
// itself, without a maximum. In the rare case that some row's sum leaves 2^+-100 they find the maxima in a pass of their own and start over
// with exp(S' - maximum). So O is never rescaled, and the steps of successive pages overlap.
//   heads of 64    as above, O in registers, four column octets per warp, the three steps of three pages behind one barrier
//   heads of 128   O in tensor memory: the sums are tcgen05 products of values (by TMA) and probabilities in shared memory, and run beside
//                  the scores of the next page and the mixing of this one
//
// The last kernel, on the CUDA cores, takes fp32, head sizes the others are not built for, and more than 64 heads.
#include <algorithm>
#include <type_traits>

#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/launch_count.h"
#include "../common/mma.cuh"
#include "../common/ptx.cuh"
#include "../common/tma_host.h"

namespace eredu {

constexpr int kPage = 16;
constexpr float kLog2e = 1.4426950408889634f;
constexpr int kMaxSplits = 8;          // portable cluster size
constexpr int kMaxHeadBlocks = 4;      // blocks of 16 heads
constexpr int kSmemLimit = 227 * 1024;
constexpr float kFar = 100.f;          // |log2| up to which exponentials are formed without subtracting a maximum

struct TalkParams {
  const void* q;           // [rows, H, dk]
  const void* k_cache;     // [pages, G, 16, dk]
  const void* v_cache;     // [pages, G, 16, dv]
  void* out;               // [rows, H, dv]
  const int* block_table;  // [B, max_pages]
  const int* seq_lens;     // [B]
  const int* cu_q;         // [B + 1] or null: q_per_seq rows each
  const void* talk;        // [H, H]
  const float* sinks;      // [H] or null
  int q_per_seq, max_pages, H, G, dk, dv, window, keep;
  float scale, softcap;
  int* status;             // where a wait that runs out is recorded
  // tensor-core kernels
  int qt;                  // queries of a CTA
  int octets;              // column octets per key / value head
  int warps;               // warps of a group
  int lanes;               // groups of a CTA
  int splits;              // CTAs of a cluster
  int group_bytes;         // shared memory of a group
};

// Visible pages of a run of queries at positions p0 .. p1: those with the first `keep` tokens, then those of the window.
struct TalkPages {
  int head, first, count;
  __device__ __forceinline__ int at(int i) const { return i < head ? i : first + i - head; }
};
__device__ __forceinline__ TalkPages talk_pages(int p0, int p1, int window, int keep) {
  TalkPages t = {0, 0, 0};
  if (p1 < 0) return t;
  if (window > 0) {
    t.head = (min(keep, p1 + 1) + kPage - 1) / kPage;
    t.first = max(t.head, max(0, p0 - window + 1) / kPage);
  }
  t.count = t.head + max(0, p1 / kPage - t.first + 1);
  return t;
}

// ---------------------------------------------------------------------------------------------- tensor cores
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// c tanh(x / (2 a)) for a pair: c - 2 c / (1 + 2^(x in)), `in` = log2(e) / a; one reciprocal serves both.
__device__ __forceinline__ void cap_pair(float& x, float& y, float in, float c) {
  const float a = 1.f + ex2(fminf(x * in, 60.f)), b = 1.f + ex2(fminf(y * in, 60.f));
  const float r = rcp(a * b) * (2.f * c);
  x = fmaf(-r, b, c);
  y = fmaf(-r, a, c);
}
// The same of one value; for any x, since 2^128 becomes infinity and its reciprocal zero.
__device__ __forceinline__ float cap_one(float x, float in, float c) { return fmaf(-2.f * c, rcp(1.f + ex2(x * in)), c); }
// x = hi + mid + lo, each exact in bf16 (truncation: 8 + 8 + 8 bits); the pieces of two values side by side.
__device__ __forceinline__ void split3(float x, float y, uint32_t& hi, uint32_t& mid, uint32_t& lo) {
  const uint32_t ux = __float_as_uint(x), uy = __float_as_uint(y);
  hi = __byte_perm(ux, uy, 0x7632);
  const float rx = x - __uint_as_float(ux & 0xFFFF0000u), ry = y - __uint_as_float(uy & 0xFFFF0000u);
  const uint32_t vx = __float_as_uint(rx), vy = __float_as_uint(ry);
  mid = __byte_perm(vx, vy, 0x7632);
  lo = __byte_perm(__float_as_uint(rx - __uint_as_float(vx & 0xFFFF0000u)), __float_as_uint(ry - __uint_as_float(vy & 0xFFFF0000u)), 0x7632);
}
__device__ __forceinline__ uint32_t pack2(float x, float y) {
  const __nv_bfloat162 t = __floats2bfloat162_rn(x, y);
  return *reinterpret_cast<const uint32_t*>(&t);
}
// The product without an order among other asm statements.
__device__ __forceinline__ void mma_pure(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void group_sync(int id, int threads) { asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(threads) : "memory"); }
__device__ __forceinline__ float ld_cluster_f32(uint32_t addr) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
  return v;
}

// Shared memory of a group, in bytes; the same arithmetic on the host and the device. Rows of keys and values are an odd number of
// 16-byte pieces long and rows of heads 8 or 24 (mod 32) floats, so that fragments load without bank conflicts.
struct TalkLayout {
  int hp;                    // heads, in whole blocks of 16
  int k_pitch, v_pitch;      // bytes of a cached row
  int k_bytes, v_bytes;      // one stage
  int s_pair, s_query;       // floats between two keys, two queries
  int s_bytes, m_bytes;
  __host__ __device__ __forceinline__ TalkLayout(int H, int G, int dk, int dv, int qt) {
    hp = (H + 15) / 16 * 16;
    k_pitch = ((dk + 15) / 16 * 2 + 1) * 16;
    v_pitch = ((dv + 15) / 16 * 2 + 1) * 16;
    k_bytes = G * kPage * k_pitch;
    v_bytes = G * kPage * v_pitch;
    s_pair = hp + 8;
    s_query = kPage * s_pair + 4;
    s_bytes = qt * s_query * 4;
    m_bytes = qt * hp * kMixPitch * 4;
  }
  static constexpr int kMixPitch = 24;   // floats of a (query, head) row of 16 mixed scores
  __host__ __device__ __forceinline__ int group() const { return 2 * (k_bytes + v_bytes) + s_bytes + m_bytes; }
  __host__ __device__ __forceinline__ int talk() const { return hp * (hp + 8) * 2; }
};

// KS, VT: 16-wide steps of the key and value sizes a warp can hold. U: column octets of a warp. The block has lanes * warps warps.
template <int KS, int VT, int U>
__global__ void __launch_bounds__(512, 1) talking_attention_kernel(TalkParams p) {
  using bf16 = __nv_bfloat16;
  extern __shared__ __align__(16) uint8_t smem[];
  pdl_launch_early();
  const TalkLayout lay(p.H, p.G, p.dk, p.dv, p.qt);
  const int tid = threadIdx.x, lane = tid & 31, quad = lane & 3, oct = lane >> 2;
  const int gi = (tid >> 5) / p.warps, gw = (tid >> 5) % p.warps;       // group, warp of it
  const int gthreads = p.warps * 32, gtid = tid - gi * gthreads;
  const int split = blockIdx.x % p.splits, b = blockIdx.y;
  const int r = p.H / p.G, columns = p.qt * r;
  uint8_t* talk_s = smem;
  uint8_t* mine = smem + lay.talk() + gi * p.group_bytes;
  uint8_t *ks = mine, *vs = ks + 2 * lay.k_bytes;
  float* sc = reinterpret_cast<float*>(vs + 2 * lay.v_bytes);
  float* mx = sc + lay.s_bytes / 4;

  // talk, and zeros wherever a fragment reads beyond the sizes
  for (int i = tid; i < (lay.talk() + p.lanes * p.group_bytes) / 16; i += blockDim.x) reinterpret_cast<uint4*>(smem)[i] = make_uint4(0, 0, 0, 0);
  __syncthreads();
  for (int i = tid; i < p.H * p.H; i += blockDim.x)
    reinterpret_cast<bf16*>(talk_s)[i / p.H * (lay.hp + 8) + i % p.H] = static_cast<const bf16*>(p.talk)[i];

  pdl_wait();
  pdl_launch_dependents();
  const int row0 = p.cu_q != nullptr ? p.cu_q[b] : b * p.q_per_seq;
  const int q_len = p.cu_q != nullptr ? p.cu_q[b + 1] - row0 : p.q_per_seq;
  const int qi0 = (blockIdx.x / p.splits) * p.qt;
  if (qi0 >= q_len) return;                                             // the whole cluster
  const int nq = min(p.qt, q_len - qi0);
  const int p0 = p.seq_lens[b] - q_len + qi0, p1 = p0 + nq - 1;
  const TalkPages pages = talk_pages(p0, p1, p.window, p.keep);
  const int* bt = p.block_table + static_cast<size_t>(b) * p.max_pages;
  // page number i of this group: the splits take contiguous shares, their groups every lanes-th page of it
  const int share = (pages.count + p.splits - 1) / p.splits;
  const int i0 = split * share + gi, i1 = min(pages.count, (split + 1) * share);
  const int n = i1 > i0 ? (i1 - i0 + p.lanes - 1) / p.lanes : 0;

  // ---- the warp's columns
  const bf16* q = static_cast<const bf16*>(p.q) + static_cast<size_t>(row0 + qi0) * p.H * p.dk;
  const int nks = (p.dk + 15) >> 4, nvt = (p.dv + 15) >> 4;
  uint32_t qf[U][KS][2];
  int kvh[U], s_off[U][2], m_off[U], col_q[U], col_h[U];
  bool on[U];
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int unit = gw * U + u;
    on[u] = unit < p.G * p.octets;
    kvh[u] = on[u] ? unit / p.octets : 0;
    const int c0 = on[u] ? (unit % p.octets) * 8 : columns;
#pragma unroll
    for (int e = 0; e < 2; ++e) {                                       // the two columns of a score fragment
      const int c = c0 + quad * 2 + e;
      s_off[u][e] = c < columns ? c / r * lay.s_query + kvh[u] * r + c % r + oct * lay.s_pair : -1;
    }
    const int c = c0 + oct;                                             // the column of a probability fragment
    col_q[u] = c < columns ? c / r : -1;
    col_h[u] = c < columns ? kvh[u] * r + c % r : 0;
    m_off[u] = (max(col_q[u], 0) * lay.hp + col_h[u]) * TalkLayout::kMixPitch + quad * 2;
    const bool real = col_q[u] >= 0 && col_q[u] < nq;
    const bf16* src = q + (static_cast<size_t>(max(col_q[u], 0)) * p.H + col_h[u]) * p.dk;
#pragma unroll
    for (int k = 0; k < KS; ++k)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int d = k * 16 + e * 8 + quad * 2;
        qf[u][k][e] = real && d < p.dk ? *reinterpret_cast<const uint32_t*>(src + d) : 0u;
      }
  }
  const float cap_c = p.softcap * kLog2e, cap_in = p.softcap > 0.f ? 2.f * kLog2e * p.scale / p.softcap : 0.f, plain = p.scale * kLog2e;

  float o[U][VT][4], m[U], l[U];
#pragma unroll
  for (int u = 0; u < U; ++u) {
    m[u] = -1e30f;
    l[u] = 0.f;
#pragma unroll
    for (int v = 0; v < VT; ++v)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[u][v][e] = 0.f;
  }

  // ---- asynchronous copies: a page's rows of all key / value heads lie in one piece
  const int kc = p.dk >> 3, vc = p.dv >> 3;                             // 16-byte pieces of a row
  const int kl2 = 32 - __clz(kc - 1), vl2 = 32 - __clz(vc - 1);         // threads per row: the next power of two
  auto load = [&](const void* cache, uint8_t* dst, int pitch, int pieces, int l2, int i) {
    const size_t page = bt[pages.at(i0 + i * p.lanes)];
    const uint4* src = static_cast<const uint4*>(cache) + page * (p.G * kPage) * pieces;
    const int c = gtid & ((1 << l2) - 1);
    if (c >= pieces) return;
    for (int row = gtid >> l2; row < p.G * kPage; row += gthreads >> l2)
      cp_async16(dst + row * pitch + c * 16, src + static_cast<size_t>(row) * pieces + c, 16);
  };
  auto load_k = [&](int i) {
    if (i < n) load(p.k_cache, ks + (i & 1) * lay.k_bytes, lay.k_pitch, kc, kl2, i);
  };
  auto load_v = [&](int i) {
    if (i < n) load(p.v_cache, vs + (i & 1) * lay.v_bytes, lay.v_pitch, vc, vl2, i);
  };

  auto score = [&](int i) {
    const uint32_t base = smem_u32(ks + (i & 1) * lay.k_bytes) + (lane & 15) * lay.k_pitch + (lane >> 4) * 16;
    float s[U][4];
#pragma unroll
    for (int u = 0; u < U; ++u) s[u][0] = s[u][1] = s[u][2] = s[u][3] = 0.f;
#pragma unroll
    for (int k = 0; k < KS; ++k) {
      if (k >= nks) break;
      uint32_t a0, a1, a2, a3;
#pragma unroll
      for (int u = 0; u < U; ++u) {
        if (!on[u]) break;
        if (u == 0 || kvh[u] != kvh[u - 1]) ldsm_x4(base + kvh[u] * (kPage * lay.k_pitch) + k * 32, a0, a1, a2, a3);
        mma16816(s[u], a0, a1, a2, a3, qf[u][k][0], qf[u][k][1]);
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (!on[u]) break;
      if (p.softcap > 0.f) {
        cap_pair(s[u][0], s[u][1], cap_in, cap_c);
        cap_pair(s[u][2], s[u][3], cap_in, cap_c);
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) s[u][e] *= plain;
      }
#pragma unroll
      for (int e = 0; e < 2; ++e)
        if (s_off[u][e] >= 0) {
          sc[s_off[u][e]] = s[u][e];
          sc[s_off[u][e] + 8 * lay.s_pair] = s[u][2 + e];
        }
    }
  };

  const int blocks = lay.hp >> 4;
  const uint32_t talk_a = smem_u32(talk_s) + (lane & 15) * (lay.hp + 8) * 2 + (lane >> 4) * 16;
  auto mix = [&]() {
    for (int t = gw; t < 2 * p.qt; t += p.warps) {                      // eight keys of a query
      const int qq = t >> 1, k0 = (t & 1) * 8;
      const float* src = sc + qq * lay.s_query + (k0 + oct) * lay.s_pair + quad * 2;
      float acc[kMaxHeadBlocks][4];
#pragma unroll
      for (int h = 0; h < kMaxHeadBlocks; ++h) acc[h][0] = acc[h][1] = acc[h][2] = acc[h][3] = 0.f;
#pragma unroll
      for (int g = 0; g < kMaxHeadBlocks; ++g) {
        if (g >= blocks) break;
        const float2 x = *reinterpret_cast<const float2*>(src + g * 16), y = *reinterpret_cast<const float2*>(src + g * 16 + 8);
        uint32_t h0, h1, m0, m1, l0, l1;
        split3(x.x, x.y, h0, m0, l0);
        split3(y.x, y.y, h1, m1, l1);
#pragma unroll
        for (int h = 0; h < kMaxHeadBlocks; ++h) {
          if (h >= blocks) break;
          uint32_t a0, a1, a2, a3;
          ldsm_x4(talk_a + h * 16 * (lay.hp + 8) * 2 + g * 32, a0, a1, a2, a3);
          mma16816(acc[h], a0, a1, a2, a3, l0, l1);
          mma16816(acc[h], a0, a1, a2, a3, m0, m1);
          mma16816(acc[h], a0, a1, a2, a3, h0, h1);
        }
      }
#pragma unroll
      for (int h = 0; h < kMaxHeadBlocks; ++h) {
        if (h >= blocks) break;
        float* dst = mx + (qq * lay.hp + h * 16 + oct) * TalkLayout::kMixPitch + k0 + quad * 2;
        *reinterpret_cast<float2*>(dst) = make_float2(acc[h][0], acc[h][1]);
        *reinterpret_cast<float2*>(dst + 8 * TalkLayout::kMixPitch) = make_float2(acc[h][2], acc[h][3]);
      }
    }
  };

  auto combine = [&](int i) {
    const int key0 = pages.at(i0 + i * p.lanes) * kPage;
    // every query sees every key of the page
    const bool inner = key0 + kPage - 1 <= p0 && (p.window <= 0 || p1 - key0 < p.window || key0 + kPage <= p.keep);
    uint32_t pf[U][2];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (!on[u]) break;
      const float2 x = *reinterpret_cast<const float2*>(mx + m_off[u]), y = *reinterpret_cast<const float2*>(mx + m_off[u] + 8);
      float s[4] = {x.x, x.y, y.x, y.y};
      if (!inner) {
        const int pos = p0 + max(col_q[u], 0);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int key = key0 + quad * 2 + (e & 1) + (e >> 1) * 8;
          if (key > pos || (p.window > 0 && pos - key >= p.window && key >= p.keep)) s[e] = -INFINITY;
        }
      }
      float top = fmaxf(fmaxf(s[0], s[1]), fmaxf(s[2], s[3]));
      top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, 1));
      top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, 2));
      // the reference point moves only when a score exceeds it by more than 2^8
      if (__any_sync(0xffffffffu, top > m[u] + 8.f)) {
        const float next = fmaxf(m[u], top), corr = ex2(m[u] - next);
        m[u] = next;
        l[u] *= corr;
        const float c0 = __shfl_sync(0xffffffffu, corr, quad * 8), c1 = __shfl_sync(0xffffffffu, corr, quad * 8 + 4);
#pragma unroll
        for (int v = 0; v < VT; ++v) {
          o[u][v][0] *= c0;
          o[u][v][1] *= c1;
          o[u][v][2] *= c0;
          o[u][v][3] *= c1;
        }
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) s[e] = ex2(s[e] - m[u]);
      l[u] += (s[0] + s[1]) + (s[2] + s[3]);
      pf[u][0] = pack2(s[0], s[1]);
      pf[u][1] = pack2(s[2], s[3]);
    }
    // matrix j of a quadruple: keys 8 (j >> 1) .., value dims 8 (j & 1) ..
    const uint32_t base = smem_u32(vs + (i & 1) * lay.v_bytes) + ((lane & 7) + (lane >> 4) * 8) * lay.v_pitch + ((lane >> 3) & 1) * 16;
#pragma unroll
    for (int v = 0; v < VT; ++v) {
      if (v >= nvt) break;
      uint32_t a0, a1, a2, a3;
#pragma unroll
      for (int u = 0; u < U; ++u) {
        if (!on[u]) break;
        if (u == 0 || kvh[u] != kvh[u - 1]) ldsm_x4_t(base + kvh[u] * (kPage * lay.v_pitch) + v * 32, a0, a1, a2, a3);
        mma16816(o[u][v], a0, a1, a2, a3, pf[u][0], pf[u][1]);
      }
    }
  };

  // ---- pages. Between the barriers of page i: its scores beside the sums of page i - 1, then its mixing. Keys are fetched two pages
  // ahead, values one: their buffers are free once every warp has passed the barrier behind their last use.
  const int bar = 1 + gi;
  load_k(0);
  load_v(0);
  cp_async_commit();
  load_k(1);
  cp_async_commit();
  cp_async_wait<1>();
  __syncthreads();                                                      // talk and the zeros, too
  if (n > 0) {
    for (int i = 0; i < n; ++i) {
      score(i);
      if (i > 0) combine(i - 1);
      group_sync(bar, gthreads);
      load_k(i + 2);
      load_v(i + 1);
      cp_async_commit();
      mix();
      cp_async_wait<1>();                                               // keys i + 1 (and values i) are there
      group_sync(bar, gthreads);
    }
    cp_async_wait<0>();
    combine(n - 1);
  }
#pragma unroll
  for (int u = 0; u < U; ++u) {
    l[u] += __shfl_xor_sync(0xffffffffu, l[u], 1);
    l[u] += __shfl_xor_sync(0xffffffffu, l[u], 2);
  }

  bf16* out = static_cast<bf16*>(p.out) + static_cast<size_t>(row0 + qi0) * p.H * p.dv;
  if (p.lanes * p.splits == 1) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (!on[u]) break;
      const float sink = p.sinks != nullptr ? p.sinks[col_h[u]] * kLog2e : -INFINITY;
      const float top = fmaxf(m[u], sink), e = ex2(m[u] - top), sum = l[u] * e + ex2(sink - top);
      const float f = sum > 0.f ? e / sum : 0.f;
      const float f0 = __shfl_sync(0xffffffffu, f, quad * 8), f1 = __shfl_sync(0xffffffffu, f, quad * 8 + 4);
      const int at = col_q[u] >= 0 && col_q[u] < nq ? (col_q[u] * p.H + col_h[u]) * p.dv : -1;
      const int at0 = __shfl_sync(0xffffffffu, at, quad * 8), at1 = __shfl_sync(0xffffffffu, at, quad * 8 + 4);
#pragma unroll
      for (int v = 0; v < VT; ++v) {
        if (v >= nvt) break;
#pragma unroll
        for (int e2 = 0; e2 < 2; ++e2) {
          const int d = v * 16 + e2 * 8 + oct;
          if (d >= p.dv) continue;
          if (at0 >= 0) out[at0 + d] = __float2bfloat16(o[u][v][e2 * 2] * f0);
          if (at1 >= 0) out[at1 + d] = __float2bfloat16(o[u][v][e2 * 2 + 1] * f1);
        }
      }
    }
    return;
  }

  // ---- partial results of the groups and of the cluster's CTAs: O [lanes][qt H][dv], then (m, l) [lanes][qt H][2], then the weights of
  // all partials [splits lanes][qt H], over the buffers of the pages
  const int rows = p.qt * p.H;
  float* part = reinterpret_cast<float*>(smem + lay.talk());
  float* ml = part + p.lanes * rows * p.dv;
  float* weight = ml + p.lanes * rows * 2;
  __syncthreads();
#pragma unroll
  for (int u = 0; u < U; ++u) {
    if (!on[u]) break;
    const int row = col_q[u] >= 0 ? col_q[u] * p.H + col_h[u] : -1;
    if (quad == 0 && row >= 0) {
      ml[(gi * rows + row) * 2] = m[u];
      ml[(gi * rows + row) * 2 + 1] = l[u];
    }
    const int at0 = __shfl_sync(0xffffffffu, row, quad * 8), at1 = __shfl_sync(0xffffffffu, row, quad * 8 + 4);
#pragma unroll
    for (int v = 0; v < VT; ++v) {
      if (v >= nvt) break;
#pragma unroll
      for (int e2 = 0; e2 < 2; ++e2) {
        const int d = v * 16 + e2 * 8 + oct;
        if (d >= p.dv) continue;
        if (at0 >= 0) part[(gi * rows + at0) * p.dv + d] = o[u][v][e2 * 2];
        if (at1 >= 0) part[(gi * rows + at1) * p.dv + d] = o[u][v][e2 * 2 + 1];
      }
    }
  }
  if (p.splits > 1) {
    cluster_arrive_release();
    cluster_wait_acquire();
  } else {
    __syncthreads();
  }
  const uint32_t ml_a = smem_u32(ml), part_a = smem_u32(part);
  for (int row = tid; row < nq * p.H; row += blockDim.x) {
    const float sink = p.sinks != nullptr ? p.sinks[row % p.H] * kLog2e : -INFINITY;
    float top = sink;
    for (int s = 0; s < p.splits; ++s)
      for (int g = 0; g < p.lanes; ++g) top = fmaxf(top, ld_cluster_f32(mapa_shared(ml_a + (g * rows + row) * 8, s)));
    float sum = ex2(sink - top);
    for (int s = 0; s < p.splits; ++s)
      for (int g = 0; g < p.lanes; ++g) {
        const uint32_t a = mapa_shared(ml_a + (g * rows + row) * 8, s);
        const float w = ex2(ld_cluster_f32(a) - top);
        sum += w * ld_cluster_f32(a + 4);
        weight[(s * p.lanes + g) * rows + row] = w;
      }
    const float inv = sum > 0.f ? 1.f / sum : 0.f;
    for (int s = 0; s < p.splits * p.lanes; ++s) weight[s * rows + row] *= inv;
  }
  __syncthreads();
  for (int i = split * blockDim.x + tid; i < nq * p.H * p.dv; i += p.splits * blockDim.x) {
    const int row = i / p.dv;
    float v = 0.f;
    for (int s = 0; s < p.splits; ++s)
      for (int g = 0; g < p.lanes; ++g)
        v = fmaf(weight[(s * p.lanes + g) * rows + row], ld_cluster_f32(mapa_shared(part_a + (g * rows * p.dv + i) * 4, s)), v);
    out[i] = __float2bfloat16(v);
  }
  if (p.splits > 1) {                                                   // nobody reads this CTA's shared memory any more
    cluster_arrive_release();
    cluster_wait_acquire();
  }
}

// How a step of at most `rows` queries per sequence is cut; qt = 0: this kernel does not take the sizes.
struct TalkPlan {
  int qt = 0, octets = 0, units = 0, per_warp = 0, warps = 0, lanes = 1, group_bytes = 0, smem = 0;
};
static TalkPlan talk_plan(int H, int G, int dk, int dv, int rows, bool decode) {
  TalkPlan best;
  if (G <= 0 || H % G != 0 || H > 16 * kMaxHeadBlocks || dk <= 0 || dv <= 0 || dk > 128 || dv > 128 || dk % 8 != 0 || dv % 8 != 0) return best;
  const int r = H / G, most = dk <= 64 && dv <= 64 ? 4 : 2;
  for (int qt = decode ? rows : 32; qt >= 1; qt = decode ? qt - 1 : qt / 2) {
    if (!decode && qt > 1 && qt / 2 >= rows) continue;
    TalkPlan t;
    t.qt = qt;
    t.octets = (qt * r + 7) / 8;
    t.units = G * t.octets;
    t.per_warp = t.units <= 16 ? 1 : t.units <= 32 ? 2 : t.units <= 64 ? 4 : 99;
    if (t.per_warp > most) continue;
    t.warps = (t.units + t.per_warp - 1) / t.per_warp;
    const TalkLayout lay(H, G, dk, dv, qt);
    t.group_bytes = lay.group();
    if (decode)
      while (t.lanes < 8 && (t.lanes + 1) * t.warps <= 16 && lay.talk() + (t.lanes + 1) * t.group_bytes <= kSmemLimit) ++t.lanes;
    // the partial results of the last phase lie over the buffers
    const int part = decode ? t.lanes * qt * H * (dv + 2 + kMaxSplits) * 4 : 0;
    t.smem = lay.talk() + std::max(t.lanes * t.group_bytes, (part + 15) / 16 * 16);
    if (t.smem > kSmemLimit) continue;
    return t;
  }
  return best;
}

template <int KS, int VT, int U>
static cudaError_t launch_talking(const TalkParams& p, dim3 grid, int threads, int smem, cudaStream_t stream) {
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(talking_attention_kernel<KS, VT, U>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemLimit);
    if (e != cudaSuccess) return e;
    configured = true;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = dim3(threads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  int n = 0;
  if (pdl_enabled()) {
    attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[n++].val.programmaticStreamSerializationAllowed = 1;
  }
  if (p.splits > 1) {
    attr[n].id = cudaLaunchAttributeClusterDimension;
    attr[n].val.clusterDim.x = p.splits;
    attr[n].val.clusterDim.y = 1;
    attr[n++].val.clusterDim.z = 1;
  }
  cfg.attrs = attr;
  cfg.numAttrs = n;
  return cudaLaunchKernelEx(&cfg, talking_attention_kernel<KS, VT, U>, p);
}

// ---------------------------------------------------------------------------------------------- prompts
// Layout of a CTA of the kernel below, in bytes; the pitches as in TalkLayout, rows of 16 probabilities 48 bytes long. Scores and
// probabilities have two buffers.
struct PromptLayout {
  TalkLayout t;
  int p_bytes;
  static constexpr int kProbPitch = 48;
  __host__ __device__ __forceinline__ PromptLayout(int H, int G, int d, int qt) : t(H, G, d, d, qt), p_bytes(qt * t.hp * kProbPitch) {}
  __host__ __device__ __forceinline__ int refs() const { return p_rows() * 4; }
  __host__ __device__ __forceinline__ int p_rows() const { return p_bytes / kProbPitch; }
  __host__ __device__ __forceinline__ int total() const { return t.talk() + 2 * (t.k_bytes + t.v_bytes + t.s_bytes + p_bytes) + refs(); }
};

// Heads of 64; HB blocks of 16 heads; NT (query, eight keys) products of the mix step per warp. A warp holds kUnits column octets of one
// key / value head.
constexpr int kUnits = 4, kPromptWarps = 8;

template <int HB, int NT>
__global__ void __launch_bounds__(32 * kPromptWarps, 1) talking_prompt_kernel(TalkParams p) {
  using bf16 = __nv_bfloat16;
  constexpr int D = 64, U = kUnits, KS = D / 16, VT = D / 16, PIECES = D / 8, PITCH = (PIECES + 1) * 16;
  constexpr int HP = 16 * HB, SP = HP + 8, SQ = kPage * SP + 4, PP = PromptLayout::kProbPitch;
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ int far_row;
  pdl_launch_early();
  const PromptLayout lay(p.H, p.G, D, p.qt);
  const int tid = threadIdx.x, lane = tid & 31, quad = lane & 3, oct = lane >> 2, gw = tid >> 5, threads = blockDim.x, nwarps = threads >> 5;
  const int b = blockIdx.y, r = p.H / p.G, columns = p.qt * r;
  uint8_t *ks = smem + lay.t.talk(), *vs = ks + 2 * lay.t.k_bytes;
  float* sc = reinterpret_cast<float*>(vs + 2 * lay.t.v_bytes);
  uint8_t* ps = reinterpret_cast<uint8_t*>(sc) + 2 * lay.t.s_bytes;
  float* ref = reinterpret_cast<float*>(ps + 2 * lay.p_bytes);          // -c of every (query, head)
  const int s_stage = lay.t.s_bytes / 4, p_stage = lay.p_bytes, kv_stage = lay.t.k_bytes;

  for (int i = tid; i < lay.total() / 16; i += threads) reinterpret_cast<uint4*>(smem)[i] = make_uint4(0, 0, 0, 0);
  __syncthreads();
  for (int i = tid; i < p.H * p.H; i += threads) reinterpret_cast<bf16*>(smem)[i / p.H * (HP + 8) + i % p.H] = static_cast<const bf16*>(p.talk)[i];

  pdl_wait();
  pdl_launch_dependents();
  const int row0 = p.cu_q != nullptr ? p.cu_q[b] : b * p.q_per_seq;
  const int q_len = p.cu_q != nullptr ? p.cu_q[b + 1] - row0 : p.q_per_seq;
  const int qi0 = blockIdx.x * p.qt;
  if (qi0 >= q_len) return;
  const int nq = min(p.qt, q_len - qi0);
  const int p0 = p.seq_lens[b] - q_len + qi0, p1 = p0 + nq - 1;
  const TalkPages pages = talk_pages(p0, p1, p.window, p.keep);
  const int* bt = p.block_table + static_cast<size_t>(b) * p.max_pages;
  const int n = pages.count;
  if (n <= 0) return;

  // ---- the warp's columns: one key / value head, U octets side by side; columns beyond the last query are zeros that nobody reads
  const int g = gw * U / p.octets, o0 = gw * U % p.octets;
  uint32_t qf[U][KS][2];
  int s_off[U][2];
#pragma unroll
  for (int u = 0; u < U; ++u) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int c = (o0 + u) * 8 + quad * 2 + e;
      s_off[u][e] = c < columns ? c / r * SQ + g * r + c % r + oct * SP : -1;
    }
    const int c = (o0 + u) * 8 + oct, cq = c / r;
    const bf16* src = static_cast<const bf16*>(p.q) + (static_cast<size_t>(row0 + qi0 + cq) * p.H + g * r + c % r) * D + quad * 2;
#pragma unroll
    for (int k = 0; k < KS; ++k)
#pragma unroll
      for (int e = 0; e < 2; ++e) qf[u][k][e] = cq < nq ? *reinterpret_cast<const uint32_t*>(src + k * 16 + e * 8) : 0u;
  }
  // rows of probabilities as a fragment of two octets reads them: lanes 0 - 7 and 8 - 15 the two halves of the first one's keys
  uint32_t p_addr[U / 2];
#pragma unroll
  for (int u = 0; u < U / 2; ++u) {
    const int c = min((o0 + 2 * u + (lane >> 4)) * 8 + (lane & 7), columns - 1);
    p_addr[u] = smem_u32(ps) + (c / r * HP + g * r + c % r) * PP + ((lane >> 3) & 1) * 16;
  }
  const uint32_t k_addr = smem_u32(ks) + (g * kPage + (lane & 15)) * PITCH + (lane >> 4) * 16;
  const uint32_t v_addr = smem_u32(vs) + (g * kPage + (lane & 7) + (lane >> 4) * 8) * PITCH + ((lane >> 3) & 1) * 16;
  const uint32_t talk_a = smem_u32(smem) + (lane & 15) * (HP + 8) * 2 + (lane >> 4) * 16;
  const float cap_c = p.softcap * kLog2e, cap_in = 2.f * kLog2e * p.scale / p.softcap;

  // ---- asynchronous copies: a page's rows of all key / value heads lie in one piece; a thread's place in it is fixed
  const int pieces = p.G * kPage * PIECES, copies = pieces / threads;
  const uint32_t copy_dst = (tid / PIECES) * PITCH + (tid % PIECES) * 16, copy_step = threads / PIECES * PITCH;
  auto load = [&](const void* cache, uint32_t dst, int page) {
    const uint4* src = static_cast<const uint4*>(cache) + static_cast<size_t>(page) * pieces + tid;
    dst += copy_dst;
#pragma unroll 4
    for (int i = 0; i < copies; ++i) {
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
      src += threads;
      dst += copy_step;
    }
  };

  float o[U][VT][4], l[NT][HB][2];
  auto score = [&](int buf) {
    float s[U][4];
#pragma unroll
    for (int u = 0; u < U; ++u) s[u][0] = s[u][1] = s[u][2] = s[u][3] = 0.f;
    const uint32_t base = k_addr + buf * kv_stage;
    uint32_t a[2][4];
    ldsm_x4(base, a[0][0], a[0][1], a[0][2], a[0][3]);
#pragma unroll
    for (int k = 0; k < KS; ++k) {
      uint32_t* c = a[k & 1];
      uint32_t* f = a[(k + 1) & 1];
      if (k + 1 < KS) ldsm_x4(base + (k + 1) * 32, f[0], f[1], f[2], f[3]);
#pragma unroll
      for (int u = 0; u < U; ++u) mma_pure(s[u], c[0], c[1], c[2], c[3], qf[u][k][0], qf[u][k][1]);
    }
    float* dst = sc + buf * s_stage;
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[u][e] = cap_one(s[u][e], cap_in, cap_c);
#pragma unroll
    for (int u = 0; u < U; ++u) {
#pragma unroll
      for (int e = 0; e < 2; ++e)
        if (s_off[u][e] >= 0) {
          dst[s_off[u][e]] = s[u][e];
          dst[s_off[u][e] + 8 * SP] = s[u][2 + e];
        }
    }
  };

  // MASK: some key of the page is hidden from some query. MAX: only the maxima, into l.
  auto mix = [&](int buf, int key0, auto masked, auto maxima) {
    constexpr bool MASK = decltype(masked)::value, MAX = decltype(maxima)::value;
    // all products side by side: their steps are long chains
    float acc[NT][HB][4];
    int row[NT];                                                        // (query, first head of the thread)
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int t = min(gw + j * nwarps, 2 * p.qt - 1);
      row[j] = (t >> 1) * HP + oct;
#pragma unroll
      for (int h = 0; h < HB; ++h) {
        acc[j][h][0] = acc[j][h][1] = ref[row[j] + h * 16];
        acc[j][h][2] = acc[j][h][3] = ref[row[j] + h * 16 + 8];
      }
    }
#pragma unroll
    for (int e = 0; e < HB; ++e) {
      uint32_t bf[NT][3][2];
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        const int t = min(gw + j * nwarps, 2 * p.qt - 1);
        const float* src = sc + buf * s_stage + (t >> 1) * SQ + ((t & 1) * 8 + oct) * SP + quad * 2 + e * 16;
        const float2 x = *reinterpret_cast<const float2*>(src), y = *reinterpret_cast<const float2*>(src + 8);
        split3(x.x, x.y, bf[j][0][0], bf[j][1][0], bf[j][2][0]);
        split3(y.x, y.y, bf[j][0][1], bf[j][1][1], bf[j][2][1]);
      }
#pragma unroll
      for (int h = 0; h < HB; ++h) {
        uint32_t a0, a1, a2, a3;
        ldsm_x4(talk_a + h * 16 * (HP + 8) * 2 + e * 32, a0, a1, a2, a3);
#pragma unroll
        for (int x = 2; x >= 0; --x)
#pragma unroll
          for (int j = 0; j < NT; ++j) mma_pure(acc[j][h], a0, a1, a2, a3, bf[j][x][0], bf[j][x][1]);
      }
    }
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int t = min(gw + j * nwarps, 2 * p.qt - 1), k0 = (t & 1) * 8;
      if constexpr (MASK) {
        const int pos = p0 + (t >> 1);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int key = key0 + k0 + quad * 2 + e;
          const bool hide = key > pos || (p.window > 0 && pos - key >= p.window && key >= p.keep);
#pragma unroll
          for (int h = 0; h < HB; ++h) {
            acc[j][h][e] = hide ? -INFINITY : acc[j][h][e];
            acc[j][h][2 + e] = hide ? -INFINITY : acc[j][h][2 + e];
          }
        }
      }
#pragma unroll
      for (int h = 0; h < HB; ++h) {
        if constexpr (MAX) {
          l[j][h][0] = fmaxf(l[j][h][0], fmaxf(acc[j][h][0], acc[j][h][1]));
          l[j][h][1] = fmaxf(l[j][h][1], fmaxf(acc[j][h][2], acc[j][h][3]));
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e) acc[j][h][e] = ex2(acc[j][h][e]);
          l[j][h][0] += acc[j][h][0] + acc[j][h][1];
          l[j][h][1] += acc[j][h][2] + acc[j][h][3];
        }
      }
    }
    if constexpr (!MAX) {
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        const int t = min(gw + j * nwarps, 2 * p.qt - 1);
        uint8_t* dst = ps + buf * p_stage + row[j] * PP + ((t & 1) * 8 + quad * 2) * 2;
#pragma unroll
        for (int h = 0; h < HB; ++h) {
          *reinterpret_cast<uint32_t*>(dst + h * 16 * PP) = pack2(acc[j][h][0], acc[j][h][1]);
          *reinterpret_cast<uint32_t*>(dst + (h * 16 + 8) * PP) = pack2(acc[j][h][2], acc[j][h][3]);
        }
      }
    }
  };

  auto combine = [&](int buf) {
    uint32_t pf[U][2];
#pragma unroll
    for (int u = 0; u < U; u += 2) ldsm_x4(p_addr[u / 2] + buf * p_stage, pf[u][0], pf[u][1], pf[u + 1][0], pf[u + 1][1]);
    const uint32_t base = v_addr + buf * kv_stage;
    uint32_t a[2][4];
    ldsm_x4_t(base, a[0][0], a[0][1], a[0][2], a[0][3]);
#pragma unroll
    for (int v = 0; v < VT; ++v) {
      uint32_t* c = a[v & 1];
      uint32_t* f = a[(v + 1) & 1];
      if (v + 1 < VT) ldsm_x4_t(base + (v + 1) * 32, f[0], f[1], f[2], f[3]);
#pragma unroll
      for (int u = 0; u < U; ++u) mma_pure(o[u][v], c[0], c[1], c[2], c[3], pf[u][0], pf[u][1]);
    }
  };

  // ---- pages. Iteration i: scores of page i + 1, mixing of page i, sums of page i - 1; keys are fetched two pages ahead, values one. What an
  // iteration writes was read before the barrier in front of it. The first one's sums are of zeros, the last one's scores are not read.
  const uint32_t ks_a = smem_u32(ks), vs_a = smem_u32(vs);
  auto page_at = [&](int i) { return bt[pages.at(min(i, n - 1))]; };
  auto walk = [&](auto maxima) {
    constexpr bool MAX = decltype(maxima)::value;
    int pg0 = page_at(0), pg1 = page_at(1), pg2 = page_at(2);
    load(p.k_cache, ks_a, pg0);
    load(p.k_cache, ks_a + kv_stage, pg1);
    cp_async_commit();
    cp_async_wait<0>();
    __syncthreads();
    score(0);
    __syncthreads();
    for (int i = 0; i < n; ++i) {
      const int pg3 = page_at(i + 3), cur = i & 1, key0 = pages.at(i) * kPage;
      const bool inner = key0 + kPage - 1 <= p0 && (p.window <= 0 || p1 - key0 < p.window || key0 + kPage <= p.keep);
      load(p.k_cache, ks_a + cur * kv_stage, pg2);
      load(p.v_cache, vs_a + cur * kv_stage, pg0);
      cp_async_commit();
      if constexpr (MAX) {
        score(cur ^ 1);
        mix(cur, key0, std::true_type(), std::true_type());
      } else if (gw < kPromptWarps / 2) {
        score(cur ^ 1);
        if (inner) mix(cur, key0, std::false_type(), std::false_type());
        else mix(cur, key0, std::true_type(), std::false_type());
        combine(cur ^ 1);
      } else {
        if (inner) mix(cur, key0, std::false_type(), std::false_type());
        else mix(cur, key0, std::true_type(), std::false_type());
        combine(cur ^ 1);
        score(cur ^ 1);
      }
      cp_async_wait<0>();
      __syncthreads();
      pg0 = pg1;
      pg1 = pg2;
      pg2 = pg3;
    }
  };
  // The l of all threads, by keys of the two halves of a page: [qt hp][2] over the probabilities of the page before the last.
  float* sums = reinterpret_cast<float*>(ps + (n & 1) * p_stage);
  auto spread = [&](auto maxima) {
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int t = min(gw + j * nwarps, 2 * p.qt - 1), qq = t >> 1;
#pragma unroll
      for (int h = 0; h < HB; ++h)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float v = l[j][h][e];
#pragma unroll
          for (int x = 1; x <= 2; x *= 2) {
            const float w = __shfl_xor_sync(0xffffffffu, v, x);
            v = decltype(maxima)::value ? fmaxf(v, w) : v + w;
          }
          if (quad == 0) sums[(qq * HP + h * 16 + e * 8 + oct) * 2 + (t & 1)] = v;
        }
    }
    __syncthreads();
  };
  auto reset = [&](float start) {
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
      for (int h = 0; h < HB; ++h) l[t][h][0] = l[t][h][1] = start;
  };
  for (int pass = 0;; ++pass) {
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
      for (int v = 0; v < VT; ++v) o[u][v][0] = o[u][v][1] = o[u][v][2] = o[u][v][3] = 0.f;
    reset(0.f);
    if (tid == 0) far_row = 0;
    walk(std::false_type());
    combine((n - 1) & 1);
    spread(std::false_type());
    if (pass > 0) break;
    for (int i = tid; i < nq * p.H; i += threads) {
      const float2 v = *reinterpret_cast<const float2*>(sums + (i / p.H * HP + i % p.H) * 2);
      if (!(v.x + v.y >= exp2f(-kFar) && v.x + v.y <= exp2f(kFar))) far_row = 1;
    }
    __syncthreads();
    if (far_row == 0) break;
    // c = the maximum of every row; probabilities start from zeros again
    reset(-INFINITY);
    walk(std::true_type());
    spread(std::true_type());
    for (int i = tid; i < p.qt * HP; i += threads) {
      const float m = fmaxf(sums[i * 2], sums[i * 2 + 1]);
      ref[i] = fabsf(m) < INFINITY ? -m : 0.f;
    }
    __syncthreads();
    for (int i = tid; i < 2 * p_stage / 16; i += threads) reinterpret_cast<uint4*>(ps)[i] = make_uint4(0, 0, 0, 0);
    __syncthreads();
  }

  bf16* out = static_cast<bf16*>(p.out) + static_cast<size_t>(row0 + qi0) * p.H * D;
#pragma unroll
  for (int u = 0; u < U; ++u) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int c = (o0 + u) * 8 + quad * 2 + e, cq = c / r, h = g * r + c % r;
      if (cq >= nq) continue;
      const float sum = sums[(cq * HP + h) * 2] + sums[(cq * HP + h) * 2 + 1];
      // the sink, in units of the row's own sum
      const float sink = p.sinks != nullptr ? fmaf(p.sinks[h], kLog2e, ref[cq * HP + h]) - __log2f(sum) : -INFINITY;
      const float f = 1.f / (sum * (1.f + ex2(fminf(sink, 120.f))));
      bf16* dst = out + (cq * p.H + h) * D + oct;
#pragma unroll
      for (int v = 0; v < VT; ++v) {
        dst[v * 16] = __float2bfloat16(o[u][v][e] * f);
        dst[v * 16 + 8] = __float2bfloat16(o[u][v][2 + e] * f);
      }
    }
  }
}

// How a run of queries is cut for the kernel above; qt = 0: it does not take the sizes.
struct PromptPlan {
  int qt = 0, octets = 0, warps = 0, smem = 0, blocks = 0, per = 0, stages = 0;   // per: products of the mix step a warp takes
};
static PromptPlan prompt_plan(int H, int G, int dk, int dv, int rows, float softcap) {
  PromptPlan best;
  if (G <= 0 || H % G != 0 || H > 64 || dk != 64 || dv != 64 || softcap <= 0.f) return best;
  for (int qt = 32; qt >= 2; qt /= 2) {
    if (qt / 2 >= rows && qt > 2) continue;
    PromptPlan t;
    t.qt = qt;
    t.octets = ((qt * (H / G) + 7) / 8 + kUnits - 1) / kUnits * kUnits;
    t.warps = G * t.octets / kUnits;
    t.blocks = H <= 16 ? 1 : H <= 32 ? 2 : 4;
    t.per = (2 * qt + t.warps - 1) / t.warps;
    const PromptLayout lay(H, G, dk, qt);
    t.smem = lay.total();
    if (t.warps > kPromptWarps || t.warps * 32 % (dk / 8) != 0 || G * kPage * (dk / 8) % (t.warps * 32) != 0 || t.per > 8 / t.blocks ||
        t.smem > kSmemLimit - 256 || lay.t.hp != 16 * t.blocks)
      continue;
    return t;
  }
  return best;
}

template <int HB, int NT>
static cudaError_t launch_prompt(const TalkParams& p, dim3 grid, const PromptPlan& t, cudaStream_t stream) {
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(talking_prompt_kernel<HB, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemLimit - 256);
    if (e != cudaSuccess) return e;
    configured = true;
  }
  return launch_pdl(talking_prompt_kernel<HB, NT>, grid, dim3(t.warps * 32), t.smem, stream, p);
}
static cudaError_t launch_prompt(const TalkParams& p, dim3 grid, const PromptPlan& t, cudaStream_t stream) {
  if (t.blocks == 1) return t.per <= 4 ? launch_prompt<1, 4>(p, grid, t, stream) : launch_prompt<1, 8>(p, grid, t, stream);
  if (t.blocks == 2) return t.per <= 2 ? launch_prompt<2, 2>(p, grid, t, stream) : launch_prompt<2, 4>(p, grid, t, stream);
  return t.per <= 1 ? launch_prompt<4, 1>(p, grid, t, stream) : launch_prompt<4, 2>(p, grid, t, stream);
}

// ---------------------------------------------------------------------------------------------- prompts, head size 128
// The same steps with the sums on tcgen05: O^T[value dim, column] of a key / value head lies in tensor memory, one product of 128 value dims x
// its columns x 16 keys a page, V as it comes (swizzled rows of keys) and P as the mix step leaves it (core matrices of 8 columns x 8 keys).
constexpr int kTcHead = 128, kTcUnits = 2;

struct PromptTcLayout {
  TalkLayout t;
  int columns;                            // of a key / value head, whole octets
  int p_head, p_bytes, kv_bytes, half;    // probabilities of a head (64 bytes apart from whole rows of banks), of a page; keys of a page, 64 dims of them
  int v_off, k_off, s_off, p_off, ref_off, sum_off, total;
  // k_stages, v_stages: pages of keys and of values that fit
  __host__ __device__ __forceinline__ PromptTcLayout(int H, int G, int qt, int octets, int k_stages, int v_stages) : t(H, G, kTcHead, kTcHead, qt) {
    columns = octets * 8;
    p_head = columns * 32 + 64;
    p_bytes = G * p_head;
    half = G * kPage * 128;
    kv_bytes = 2 * half;
    v_off = 0;                            // 1024-byte aligned
    k_off = v_stages * kv_bytes;
    s_off = k_off + k_stages * kv_bytes;
    p_off = s_off + 2 * t.s_bytes;
    ref_off = p_off + 2 * p_bytes;
    sum_off = ref_off + qt * t.hp * 4;
    total = sum_off + qt * t.hp * 8 + t.talk();
  }
};

// K-major operand in core matrices of 8 rows x 16 bytes: the two halves of K = 16 lie 128 bytes apart, groups of 8 rows 256.
__device__ __forceinline__ uint64_t umma_desc_k_core(uint32_t smem_addr) {
  return static_cast<uint64_t>((smem_addr & 0x3FFFF) >> 4) | static_cast<uint64_t>(128 >> 4) << 16 | static_cast<uint64_t>(256 >> 4) << 32 |
         static_cast<uint64_t>(1) << 46;
}
// MN-major operand, rows of 64 elements (128-byte swizzle), 16 rows: the next 64 elements `lbo` bytes on, 8 rows 1024.
__device__ __forceinline__ uint64_t umma_desc_mn_rows(uint32_t smem_addr, uint32_t lbo) {
  return static_cast<uint64_t>((smem_addr & 0x3FFFF) >> 4) | static_cast<uint64_t>(lbo >> 4) << 16 | static_cast<uint64_t>(1024 >> 4) << 32 |
         static_cast<uint64_t>(1) << 46 | static_cast<uint64_t>(2) << 61;
}

__device__ __forceinline__ void sts_f32(uint32_t addr, float v) { asm volatile("st.shared.f32 [%0], %1;" ::"r"(addr), "f"(v) : "memory"); }
__device__ __forceinline__ void sts_u32(uint32_t addr, uint32_t v) { asm volatile("st.shared.u32 [%0], %1;" ::"r"(addr), "r"(v) : "memory"); }
__device__ __forceinline__ void sts_f32x2(uint32_t addr, float x, float y) {
  asm volatile("st.shared.v2.f32 [%0], {%1, %2};" ::"r"(addr), "f"(x), "f"(y) : "memory");
}
__device__ __forceinline__ float2 lds_f32x2(uint32_t addr) {
  float2 v;
  asm volatile("ld.shared.v2.f32 {%0, %1}, [%2];" : "=f"(v.x), "=f"(v.y) : "r"(addr));
  return v;
}
// Queries of a CTA: with HB blocks of 16 heads, 256 rows of a (query, head) pair.
constexpr int tc_queries(int hb) { return 16 / hb; }

// W warps, of which each takes NT products of the mix step, and three that start the copies of keys, those of values, and the sums. NK, NV:
// stages of keys and values. tm_k, tm_v: the caches as rows of 128, boxes of 64 columns and a page's rows.
template <int HB, int W, int NK, int NV>
__global__ void __launch_bounds__(32 * (W + 3), 1)
talking_prompt_tc_kernel(const __grid_constant__ CUtensorMap tm_k, const __grid_constant__ CUtensorMap tm_v, TalkParams p) {
  using bf16 = __nv_bfloat16;
  constexpr int D = kTcHead, U = kTcUnits, KS = D / 16, QT = tc_queries(HB), THREADS = 32 * (W + 3);
  constexpr int HP = 16 * HB, SP = HP + 8, SQ = kPage * SP + 4, S_STAGE = QT * SQ * 4, NT = 2 * QT > W ? 2 * QT / W : 1;
  extern __shared__ __align__(16) uint8_t smem_raw[];
  __shared__ int far_row;
  __shared__ uint32_t tmem_slot;
  __shared__ __align__(8) uint64_t k_full[NK], k_free[NK], v_full[NV], v_free[NV], step[2], done[2];
  pdl_launch_early();
  uint8_t* smem = smem_raw + ((1024 - (smem_u32(smem_raw) & 1023)) & 1023);
  const PromptTcLayout lay(p.H, p.G, QT, p.octets, NK, NV);
  const int tid = threadIdx.x, lane = tid & 31, quad = lane & 3, oct = lane >> 2, gw = tid >> 5;
  const int b = blockIdx.y, r = p.H / p.G, columns = QT * r;
  float* ref = reinterpret_cast<float*>(smem + lay.ref_off);            // -c of every (query, head)
  float* sums = reinterpret_cast<float*>(smem + lay.sum_off);           // [QT HP][2]
  bf16* talk_s = reinterpret_cast<bf16*>(smem + lay.total - lay.t.talk());
  const int p_stage = lay.p_bytes, kv_stage = lay.kv_bytes;

  for (int i = lay.s_off / 16 + tid; i < lay.total / 16; i += THREADS) reinterpret_cast<uint4*>(smem)[i] = make_uint4(0, 0, 0, 0);
  __syncthreads();
  for (int i = tid; i < p.H * p.H; i += THREADS) talk_s[i / p.H * (HP + 8) + i % p.H] = static_cast<const bf16*>(p.talk)[i];

  pdl_wait();
  pdl_launch_dependents();
  const int row0 = p.cu_q != nullptr ? p.cu_q[b] : b * p.q_per_seq;
  const int q_len = p.cu_q != nullptr ? p.cu_q[b + 1] - row0 : p.q_per_seq;
  const int qi0 = blockIdx.x * QT;
  if (qi0 >= q_len) return;
  const int nq = min(QT, q_len - qi0);
  const int p0 = p.seq_lens[b] - q_len + qi0, p1 = p0 + nq - 1;
  const TalkPages pages = talk_pages(p0, p1, p.window, p.keep);
  const int* bt = p.block_table + static_cast<size_t>(b) * p.max_pages;
  const int n = pages.count;
  if (n <= 0) return;

  int tcols = 32;
  while (tcols < p.G * lay.columns) tcols *= 2;
  if (gw == 0) {
    tmem_alloc(&tmem_slot, tcols);
    tmem_relinquish();
  }
  if (tid == 32) {
    for (int i = 0; i < NK; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_free[i], W);
    }
    for (int i = 0; i < NV; ++i) {
      mbar_init(&v_full[i], 1);
      mbar_init(&v_free[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&step[i], W);
      mbar_init(&done[i], 1);
    }
    fence_mbar_init();
    tma_prefetch_desc(&tm_k);
    tma_prefetch_desc(&tm_v);
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = tmem_slot;
  const uint32_t base_a = smem_u32(smem), ks_a = base_a + lay.k_off, vs_a = base_a + lay.v_off, ps_a = base_a + lay.p_off, sc_a = base_a + lay.s_off;

  // ---- the warp's columns: one key / value head, U octets side by side; columns beyond the last query are zeros, their scores go into the
  // gaps between rows of heads
  const bool works = gw < W;
  const int g = works ? gw * U / p.octets : 0, o0 = gw * U % p.octets;
  uint32_t qf[U][KS][2], s_dst[U][2];
  const bool pairs = r % 2 == 0;
#pragma unroll
  for (int u = 0; u < U; ++u) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int c = (o0 + u) * 8 + quad * 2 + e;
      s_dst[u][e] = sc_a + 4 * (oct * SP + (c < columns ? c / r * SQ + g * r + c % r : HP));
    }
    const int c = (o0 + u) * 8 + oct, cq = c / r;
    const bf16* src = static_cast<const bf16*>(p.q) + (static_cast<size_t>(row0 + qi0 + cq) * p.H + g * r + c % r) * D + quad * 2;
#pragma unroll
    for (int k = 0; k < KS; ++k)
#pragma unroll
      for (int e = 0; e < 2; ++e) qf[u][k][e] = cq < nq ? *reinterpret_cast<const uint32_t*>(src + k * 16 + e * 8) : 0u;
  }
  // ---- where the warp's products of the mix step (eight keys of a query) read scores and leave probabilities; those of heads that do not
  // exist go into the gaps between heads
  const bool mixes = works && gw < 2 * QT;
  const int k_half = (gw & 1) * 8;                                      // W is even: all products of a warp are of one half of the keys
  uint32_t mix_src[NT], p_dst[NT][HB][2];
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    const int qq = (gw + j * W) >> 1;
    mix_src[j] = sc_a + 4 * (qq * SQ + (k_half + oct) * SP + quad * 2);
#pragma unroll
    for (int h = 0; h < HB; ++h)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int head = h * 16 + e * 8 + oct, c = qq * r + head % r;
        p_dst[j][h][e] = ps_a + quad * 4 + (head < p.H ? head / r * lay.p_head + (c >> 3) * 256 + k_half * 16 + (c & 7) * 16 : lay.columns * 32);
      }
  }
  // row of a key fragment; the 16-byte piece of a step is found by an exclusive or (128-byte swizzle)
  const uint32_t k_addr = ks_a + (g * kPage + (lane & 15)) * 128 + (((lane >> 4) ^ (lane & 7)) << 4);
  const uint32_t talk_a = smem_u32(talk_s) + (lane & 15) * (HP + 8) * 2 + (lane >> 4) * 16;
  const float cap_m2c = -2.f * p.softcap * kLog2e, cap_c = p.softcap * kLog2e, cap_in = 2.f * kLog2e * p.scale / p.softcap;

  float l[NT][HB][2];
  auto score = [&](int from, int buf) {
    float s[U][4];
#pragma unroll
    for (int u = 0; u < U; ++u) s[u][0] = s[u][1] = s[u][2] = s[u][3] = 0.f;
    const uint32_t base = k_addr + from * kv_stage;
    uint32_t a[KS][4];
#pragma unroll
    for (int k = 0; k < KS / 2; ++k) ldsm_x4(base ^ (k << 5), a[k][0], a[k][1], a[k][2], a[k][3]);
#pragma unroll
    for (int k = 0; k < KS; ++k) {
      const int f = k + KS / 2;                                         // fetched while step k is computed
      if (f < KS) ldsm_x4((base + lay.half) ^ (k << 5), a[f][0], a[f][1], a[f][2], a[f][3]);
#pragma unroll
      for (int u = 0; u < U; ++u) mma_pure(s[u], a[k][0], a[k][1], a[k][2], a[k][3], qf[u][k][0], qf[u][k][1]);
    }
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[u][e] = fmaf(cap_m2c, rcp(1.f + ex2(s[u][e] * cap_in)), cap_c);
    const uint32_t stage = buf * S_STAGE;
    if (pairs) {                                                        // two columns are neighbouring heads of one query
#pragma unroll
      for (int u = 0; u < U; ++u) {
        sts_f32x2(s_dst[u][0] + stage, s[u][0], s[u][1]);
        sts_f32x2(s_dst[u][0] + stage + 32 * SP, s[u][2], s[u][3]);
      }
    } else {
#pragma unroll
      for (int u = 0; u < U; ++u)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          sts_f32(s_dst[u][e] + stage, s[u][e]);
          sts_f32(s_dst[u][e] + stage + 32 * SP, s[u][2 + e]);
        }
    }
  };

  // MASK: some key of the page is hidden from some query. MAX: only the maxima, into l. REF: c is not zero.
  auto mix = [&](int buf, int p_buf, int key0, auto masked, auto maxima, auto refs) {
    constexpr bool MASK = decltype(masked)::value, MAX = decltype(maxima)::value, REF = decltype(refs)::value;
    float acc[NT][HB][4];
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int h = 0; h < HB; ++h) {
        acc[j][h][0] = acc[j][h][1] = REF ? ref[((gw + j * W) >> 1) * HP + h * 16 + oct] : 0.f;
        acc[j][h][2] = acc[j][h][3] = REF ? ref[((gw + j * W) >> 1) * HP + h * 16 + 8 + oct] : 0.f;
      }
    const uint32_t s_stage = buf * S_STAGE, stage = p_buf * p_stage;
#pragma unroll
    for (int e = 0; e < HB; ++e) {
      uint32_t bf[NT][3][2];
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        const float2 x = lds_f32x2(mix_src[j] + s_stage + e * 64), y = lds_f32x2(mix_src[j] + s_stage + e * 64 + 32);
        split3(x.x, x.y, bf[j][0][0], bf[j][1][0], bf[j][2][0]);
        split3(y.x, y.y, bf[j][0][1], bf[j][1][1], bf[j][2][1]);
      }
#pragma unroll
      for (int h = 0; h < HB; ++h) {
        uint32_t a0, a1, a2, a3;
        ldsm_x4(talk_a + h * 16 * (HP + 8) * 2 + e * 32, a0, a1, a2, a3);
#pragma unroll
        for (int x = 2; x >= 0; --x)
#pragma unroll
          for (int j = 0; j < NT; ++j) mma_pure(acc[j][h], a0, a1, a2, a3, bf[j][x][0], bf[j][x][1]);
      }
    }
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      if constexpr (MASK) {
        const int pos = p0 + ((gw + j * W) >> 1);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int key = key0 + k_half + quad * 2 + e;
          const bool hide = key > pos || (p.window > 0 && pos - key >= p.window && key >= p.keep);
#pragma unroll
          for (int h = 0; h < HB; ++h) {
            acc[j][h][e] = hide ? -INFINITY : acc[j][h][e];
            acc[j][h][2 + e] = hide ? -INFINITY : acc[j][h][2 + e];
          }
        }
      }
#pragma unroll
      for (int h = 0; h < HB; ++h) {
        if constexpr (MAX) {
          l[j][h][0] = fmaxf(l[j][h][0], fmaxf(acc[j][h][0], acc[j][h][1]));
          l[j][h][1] = fmaxf(l[j][h][1], fmaxf(acc[j][h][2], acc[j][h][3]));
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e) acc[j][h][e] = ex2(acc[j][h][e]);
          l[j][h][0] += acc[j][h][0] + acc[j][h][1];
          l[j][h][1] += acc[j][h][2] + acc[j][h][3];
        }
      }
    }
    if constexpr (!MAX) {
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int h = 0; h < HB; ++h)
#pragma unroll
          for (int e = 0; e < 2; ++e) sts_u32(p_dst[j][h][e] + stage, pack2(acc[j][h][2 * e], acc[j][h][2 * e + 1]));
    }
  };

  // ---- pages. In step i the W warps form the scores of page i + 1 and mix those of page i, in either order; a barrier of theirs ends it.
  // Three threads run beside them: keys are fetched as stages become free of scores, values as they become free of sums, and page i is summed
  // up once all warps have arrived on `step`. Probabilities of page i take the place of page i - 2 and wait for its sums (`done`). Every pass
  // over the pages completes each of these barriers once per page (values: only where there are sums); running numbers give parities.
  const uint32_t idesc = umma_idesc_bf16(D, lay.columns) | (1u << 15);  // A is MN-major
  bool ok = true;
  int k_base = 0, v_base = 0;
  auto wait_for = [&](uint64_t* bar, int parity, int code) {
    if (ok) ok = mbar_wait(bar, parity & 1, p.status, code);
  };
  // page i into its stage, the pages before it counted by `base`
  auto load = [&](const CUtensorMap* map, uint64_t* full, uint64_t* empty, int off, int stages, int x, int page) {
    const int st = x % stages, page_row = page * (p.G * kPage);
    uint8_t* dst = smem + off + st * kv_stage;
    if (x >= stages) wait_for(&empty[st], x / stages - 1, 2);
    mbar_arrive_expect_tx(&full[st], kv_stage);
    tma_load_2d(dst, map, 0, page_row, &full[st]);
    tma_load_2d(dst + lay.half, map, 64, page_row, &full[st]);
  };
  auto wait_sums = [&](int i) { wait_for(&done[(k_base + i) & 1], (k_base + i) >> 1, 3); };
  using Yes = std::true_type;
  using No = std::false_type;
  auto walk = [&](auto maxima, auto refs) {
    constexpr bool MAX = decltype(maxima)::value, REF = decltype(refs)::value;
    if (works) {
      int st = k_base % NK, parity = k_base / NK;
      auto score_next = [&](int buf) {
        wait_for(&k_full[st], parity, 1);
        score(st, buf);
        __syncwarp();
        if (lane == 0) mbar_arrive(&k_free[st]);
        if (++st == NK) {
          st = 0;
          ++parity;
        }
      };
      score_next(0);
      group_sync(1, 32 * W);
      for (int i = 0; i < n; ++i) {
        const int cur = i & 1, p_buf = (k_base + i) & 1, key0 = pages.at(i) * kPage;
        const bool inner = key0 + kPage - 1 <= p0 && (p.window <= 0 || p1 - key0 < p.window || key0 + kPage <= p.keep), more = i + 1 < n;
        if constexpr (MAX || REF) {
          if (more) score_next(cur ^ 1);
          if (i > 1) wait_sums(i - 2);
          if (mixes) mix(cur, p_buf, key0, Yes(), maxima, refs);
        } else if (gw < W / 2) {
          if (more) score_next(cur ^ 1);
          if (i > 1) wait_sums(i - 2);
          if (mixes) {
            if (inner) mix(cur, p_buf, key0, No(), No(), No());
            else mix(cur, p_buf, key0, Yes(), No(), No());
          }
        } else {
          if (i > 1) wait_sums(i - 2);
          if (mixes) {
            if (inner) mix(cur, p_buf, key0, No(), No(), No());
            else mix(cur, p_buf, key0, Yes(), No(), No());
          }
          if (more) score_next(cur ^ 1);
        }
        fence_proxy_async_smem();
        __syncwarp();
        if (lane == 0) mbar_arrive(&step[p_buf]);
        group_sync(1, 32 * W);
      }
    } else if (lane == 0 && gw == W) {
      int page = bt[pages.at(0)];
      for (int i = 0; i < n; ++i) {
        const int next = i + 1 < n ? bt[pages.at(i + 1)] : 0;
        load(&tm_k, k_full, k_free, lay.k_off, NK, k_base + i, page);
        page = next;
      }
    } else if (lane == 0 && gw == W + 1) {
      int page = MAX ? 0 : bt[pages.at(0)];
      for (int i = 0; !MAX && i < n; ++i) {
        const int next = i + 1 < n ? bt[pages.at(i + 1)] : 0;
        load(&tm_v, v_full, v_free, lay.v_off, NV, v_base + i, page);
        page = next;
      }
    } else if (lane == 0) {
      const uint64_t a_desc = umma_desc_mn_rows(vs_a, lay.half), b_desc = umma_desc_k_core(ps_a);
      for (int i = 0; i < n; ++i) {
        const int buf = (k_base + i) & 1, sv = (v_base + i) % NV;
        if constexpr (!MAX) wait_for(&v_full[sv], (v_base + i) / NV, 1);
        wait_for(&step[buf], (k_base + i) >> 1, 2);
        if constexpr (MAX) {
          mbar_arrive(&done[buf]);
        } else {                                                        // O^T += V^T P^T of page i
          tc_fence_after_sync();
          uint64_t a = a_desc + ((sv * kv_stage) >> 4), b = b_desc + ((buf * p_stage) >> 4);
          for (int h = 0; h < p.G; ++h) {
            umma_f16(tmem + h * lay.columns, a, b, idesc, i > 0 ? 1u : 0u);
            a += (kPage * 128) >> 4;
            b += lay.p_head >> 4;
          }
          umma_commit(&done[buf]);
          umma_commit(&v_free[sv]);
        }
      }
    }
    __syncwarp();
    if (works || lane == 0) wait_sums(n - 1);
    __syncwarp();
    tc_fence_after_sync();
    k_base += n;
    if (!MAX) v_base += n;
  };
  // the l of all threads, by keys of the two halves of a page
  auto spread = [&](auto maxima) {
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int h = 0; h < HB; ++h)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float v = l[j][h][e];
#pragma unroll
          for (int x = 1; x <= 2; x *= 2) {
            const float w = __shfl_xor_sync(0xffffffffu, v, x);
            v = decltype(maxima)::value ? fmaxf(v, w) : v + w;
          }
          if (quad == 0 && mixes) sums[(((gw + j * W) >> 1) * HP + h * 16 + e * 8 + oct) * 2 + (gw & 1)] = v;
        }
    __syncthreads();
  };
  auto reset = [&](float start) {
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
      for (int h = 0; h < HB; ++h) l[t][h][0] = l[t][h][1] = start;
  };
  reset(0.f);
  if (tid == 0) far_row = 0;
  walk(No(), No());
  spread(No());
  for (int i = tid; i < nq * p.H; i += THREADS) {
    const float2 v = *reinterpret_cast<const float2*>(sums + (i / p.H * HP + i % p.H) * 2);
    if (!(v.x + v.y >= exp2f(-kFar) && v.x + v.y <= exp2f(kFar))) far_row = 1;
  }
  __syncthreads();
  if (far_row != 0) {
    reset(-INFINITY);                                                   // c = the maximum of every row
    walk(Yes(), No());
    spread(Yes());
    for (int i = tid; i < QT * HP; i += THREADS) {
      const float m = fmaxf(sums[i * 2], sums[i * 2 + 1]);
      ref[i] = fabsf(m) < INFINITY ? -m : 0.f;
    }
    __syncthreads();
    reset(0.f);
    walk(No(), Yes());
    spread(No());
  }

  // ---- factor and place of every column, over the scores; then O^T, a lane per value dim
  float* factor = reinterpret_cast<float*>(smem + lay.s_off);
  int* place = reinterpret_cast<int*>(factor + p.G * lay.columns);
  for (int i = tid; i < p.G * lay.columns; i += THREADS) {
    const int c = i % lay.columns, cq = c / r, h = i / lay.columns * r + c % r;
    float f = 0.f;
    if (cq < nq) {
      const float sum = sums[(cq * HP + h) * 2] + sums[(cq * HP + h) * 2 + 1];
      // the sink, in units of the row's own sum
      const float sink = p.sinks != nullptr ? fmaf(p.sinks[h], kLog2e, ref[cq * HP + h]) - __log2f(sum) : -INFINITY;
      f = 1.f / (sum * (1.f + ex2(fminf(sink, 120.f))));
    }
    factor[i] = f;
    place[i] = cq < nq ? (cq * p.H + h) * D : -1;
  }
  __syncthreads();
  bf16* out = static_cast<bf16*>(p.out) + static_cast<size_t>(row0 + qi0) * p.H * D + (gw & 3) * 32 + lane;
  for (int c0 = works ? (gw >> 2) * 16 : 1 << 20; c0 < p.G * lay.columns; c0 += (W >> 2) * 16) {
    uint32_t v[16];
    tmem_ld16(tmem + (static_cast<uint32_t>((gw & 3) * 32) << 16) + c0, v);
    tmem_wait_ld();
#pragma unroll
    for (int c = 0; c < 16; ++c)
      if (place[c0 + c] >= 0) out[place[c0 + c]] = __float2bfloat16(__uint_as_float(v[c]) * factor[c0 + c]);
  }
  tc_fence_before_sync();
  __syncthreads();
  if (gw == 0) {
    tc_fence_after_sync();
    tmem_dealloc(tmem, tcols);
  }
}

static PromptPlan prompt_tc_plan(int H, int G, int dk, int dv, float softcap) {
  PromptPlan t;
  if (G <= 0 || H % G != 0 || H > 64 || dk != kTcHead || dv != kTcHead || softcap <= 0.f) return t;
  t.blocks = H <= 16 ? 1 : H <= 32 ? 2 : 4;
  const int qt = tc_queries(t.blocks);
  t.octets = ((qt * (H / G) + 7) / 8 + kTcUnits - 1) / kTcUnits * kTcUnits;
  t.warps = G * t.octets / kTcUnits;
  for (int stages : {4, 3}) {             // of keys; values have as many, or two where the keys have three
    const PromptTcLayout lay(H, G, qt, t.octets, stages, stages == 4 ? 4 : 2);
    t.smem = lay.total + 1024;
    t.stages = stages;
    // octets * 8 columns are the N of a product; a page's rows are one box
    if ((t.warps == 8 || t.warps == 16) && t.octets <= 32 && G * kPage <= 256 && lay.t.hp == 16 * t.blocks && t.smem <= kSmemLimit - 256) {
      t.qt = qt;
      break;
    }
  }
  return t;
}

template <int HB, int W, int NK, int NV>
static cudaError_t launch_prompt_tc(const CUtensorMap& tm_k, const CUtensorMap& tm_v, const TalkParams& p, dim3 grid, const PromptPlan& t, cudaStream_t stream) {
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(talking_prompt_tc_kernel<HB, W, NK, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemLimit - 256);
    if (e != cudaSuccess) return e;
    configured = true;
  }
  return launch_pdl(talking_prompt_tc_kernel<HB, W, NK, NV>, grid, dim3((W + 3) * 32), t.smem, stream, tm_k, tm_v, p);
}
// A cudaError_t, or a negative number where a tensor map cannot be made.
static int launch_prompt_tc(const TalkParams& p, int pages, dim3 grid, const PromptPlan& t, cudaStream_t stream) {
  CUtensorMap tm_k, tm_v;
  const uint64_t rows = static_cast<uint64_t>(pages) * p.G * kPage;
  int r = make_tma_2d(&tm_k, p.k_cache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, rows, kTcHead, kTcHead, p.G * kPage, 64);
  if (r != 0) return -100 - r;
  r = make_tma_2d(&tm_v, p.v_cache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, rows, kTcHead, kTcHead, p.G * kPage, 64);
  if (r != 0) return -200 - r;
  cudaError_t e;
#define ER_TC(HB_, W_) \
  (t.stages == 4 ? launch_prompt_tc<HB_, W_, 4, 4>(tm_k, tm_v, p, grid, t, stream) : launch_prompt_tc<HB_, W_, 3, 2>(tm_k, tm_v, p, grid, t, stream))
  if (t.blocks == 1) e = t.warps == 8 ? ER_TC(1, 8) : ER_TC(1, 16);
  else if (t.blocks == 2) e = t.warps == 8 ? ER_TC(2, 8) : ER_TC(2, 16);
  else e = t.warps == 8 ? ER_TC(4, 8) : ER_TC(4, 16);
#undef ER_TC
  return static_cast<int>(e);
}

// ---------------------------------------------------------------------------------------------- CUDA cores
constexpr int kKeys = 32;

// One CTA per query: groups of 32 visible keys, first the scores of all heads, then their mixture, then a running softmax per head.
template <typename T>
__global__ void __launch_bounds__(256) talking_simt_kernel(TalkParams p) {
  extern __shared__ __align__(16) float fs[];
  float* q = fs;                            // [H dk]
  float* o = q + p.H * p.dk;                // [H dv]
  float* sc = o + p.H * p.dv;               // [32][H + 1]
  float* mx = sc + kKeys * (p.H + 1);       // [H][33]
  float* m = mx + p.H * (kKeys + 1);        // [H], then l and the factor of a step
  float *l = m + p.H, *corr = l + p.H;
  __shared__ int rows[kKeys];               // page * 16 + offset
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.y, tid = threadIdx.x, lane = tid & 31;
  const int row0 = p.cu_q != nullptr ? p.cu_q[b] : b * p.q_per_seq;
  const int q_len = p.cu_q != nullptr ? p.cu_q[b + 1] - row0 : p.q_per_seq;
  if (static_cast<int>(blockIdx.x) >= q_len) return;
  const int pos = p.seq_lens[b] - q_len + blockIdx.x, r = p.H / p.G;
  const int* bt = p.block_table + static_cast<size_t>(b) * p.max_pages;
  const T* qg = static_cast<const T*>(p.q) + static_cast<size_t>(row0 + blockIdx.x) * p.H * p.dk;
  const T* talk = static_cast<const T*>(p.talk);
  for (int i = tid; i < p.H * p.dk; i += 256) q[i] = to_f32(qg[i]);
  for (int i = tid; i < p.H * p.dv; i += 256) o[i] = 0.f;
  for (int i = tid; i < p.H; i += 256) {
    m[i] = p.sinks != nullptr ? p.sinks[i] : -INFINITY;
    l[i] = p.sinks != nullptr ? 1.f : 0.f;
  }
  // visible keys in order: `head` first ones, then from `first` on
  const int head = p.window > 0 ? min(p.keep, pos + 1) : 0, first = p.window > 0 ? max(head, pos - p.window + 1) : 0;
  const int total = head + max(0, pos - first + 1);
  for (int k0 = 0; k0 < total; k0 += kKeys) {
    const int n = min(kKeys, total - k0);
    __syncthreads();
    if (tid < n) {
      const int i = k0 + tid, key = i < head ? i : first + i - head;
      rows[tid] = bt[key >> 4] * 16 + (key & 15);
    }
    __syncthreads();
    for (int i = tid; i < p.H * kKeys; i += 256) {
      const int h = i / kKeys, j = i % kKeys;
      if (j >= n) continue;
      const T* k = static_cast<const T*>(p.k_cache) + ((static_cast<size_t>(rows[j] >> 4) * p.G + h / r) * 16 + (rows[j] & 15)) * p.dk;
      float s = 0.f;
      for (int d = 0; d < p.dk; ++d) s = fmaf(q[h * p.dk + d], to_f32(k[d]), s);
      s *= p.scale;
      sc[j * (p.H + 1) + h] = p.softcap > 0.f ? p.softcap * tanhf(s / p.softcap) : s;
    }
    __syncthreads();
    for (int i = tid; i < p.H * kKeys; i += 256) {
      const int h = i / kKeys, j = i % kKeys;
      float s = -INFINITY;
      if (j < n) {
        s = 0.f;
        for (int g = 0; g < p.H; ++g) s = fmaf(to_f32(talk[h * p.H + g]), sc[j * (p.H + 1) + g], s);
      }
      mx[h * (kKeys + 1) + j] = s;
    }
    __syncthreads();
    for (int h = tid >> 5; h < p.H; h += 8) {
      const float s = mx[h * (kKeys + 1) + lane];
      float top = s;
#pragma unroll
      for (int x = 16; x > 0; x >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, x));
      const float next = fmaxf(m[h], top), e = expf(s - next), sum = warp_sum_f32(e);
      mx[h * (kKeys + 1) + lane] = e;
      __syncwarp();
      if (lane == 0) {
        corr[h] = expf(m[h] - next);
        l[h] = l[h] * corr[h] + sum;
        m[h] = next;
      }
    }
    __syncthreads();
    for (int i = tid; i < p.H * p.dv; i += 256) {
      const int h = i / p.dv, d = i - h * p.dv;
      float v = o[i] * corr[h];
      for (int j = 0; j < n; ++j)
        v = fmaf(mx[h * (kKeys + 1) + j],
                 to_f32(static_cast<const T*>(p.v_cache)[((static_cast<size_t>(rows[j] >> 4) * p.G + h / r) * 16 + (rows[j] & 15)) * p.dv + d]), v);
      o[i] = v;
    }
  }
  __syncthreads();
  T* out = static_cast<T*>(p.out) + static_cast<size_t>(row0 + blockIdx.x) * p.H * p.dv;
  for (int i = tid; i < p.H * p.dv; i += 256) out[i] = from_f32<T>(l[i / p.dv] > 0.f ? o[i] / l[i / p.dv] : 0.f);
}

static TalkParams talk_params(const void* q, const void* k_cache, const void* v_cache, void* out, const int* block_table, const int* seq_lens,
                              const int* cu_q, const void* talk, const float* sinks, int q_per_seq, int max_pages, int H, int G, int dk,
                              int dv, int window, int keep, float scale, float softcap) {
  TalkParams p = {};
  p.q = q;
  p.k_cache = k_cache;
  p.v_cache = v_cache;
  p.out = out;
  p.block_table = block_table;
  p.seq_lens = seq_lens;
  p.cu_q = cu_q;
  p.talk = talk;
  p.sinks = sinks;
  p.q_per_seq = q_per_seq;
  p.max_pages = max_pages;
  p.H = H;
  p.G = G;
  p.dk = dk;
  p.dv = dv;
  p.window = window;
  p.keep = window > 0 ? keep : 0;
  p.scale = scale;
  p.softcap = softcap;
  return p;
}

constexpr int kDecodeRows = 8;   // up to this many queries per sequence are cut as decode steps

}  // namespace eredu

using namespace eredu;

// 1 when the tensor-core kernel takes steps of at most `rows` queries per sequence of these sizes.
extern "C" int eredu_talking_fits(int H, int G, int dk, int dv, int rows) {
  return talk_plan(H, G, dk, dv, rows, false).qt > 0 && talk_plan(H, G, dk, dv, std::min(rows, kDecodeRows), true).qt > 0;
}

// bf16. q [rows, H, dk] (rows of sequence b: cu_q[b] .. cu_q[b + 1], or q_per_seq each; at most max_rows), its last positions; caches
// [pages, G, 16, dk or dv]; talk [H, H] bf16; sinks fp32 [H] or null; window 0: all earlier keys, else the newest `window` and the first
// `keep`. splits <= 8: CTAs that share a sequence's keys in a decode step (cu_q null).
extern "C" int eredu_talking_attention(const void* q, const void* k_cache, const void* v_cache, void* out, const int* block_table,
                                       const int* seq_lens, const int* cu_q, const void* talk, const float* sinks, int batch, int q_per_seq,
                                       int max_rows, int max_pages, int H, int G, int dk, int dv, int window, int keep, int splits, int pages,
                                       float scale, float softcap, int* status, cudaStream_t stream) {
  if (batch <= 0 || max_rows <= 0) return 0;
  if (window < 0 || keep < 0 || splits < 1 || splits > kMaxSplits || batch > 65535) return -1;
  const bool decode = cu_q == nullptr && max_rows <= kDecodeRows;
  TalkParams p = talk_params(q, k_cache, v_cache, out, block_table, seq_lens, cu_q, talk, sinks, q_per_seq, max_pages, H, G, dk, dv, window,
                             keep, scale, softcap);
  p.status = status;
  if (!decode) {
    const bool wide = dk == kTcHead;
    const PromptPlan t = wide ? prompt_tc_plan(H, G, dk, dv, softcap) : prompt_plan(H, G, dk, dv, max_rows, softcap);
    if (t.qt > 0) {
      p.qt = t.qt;
      p.octets = t.octets;
      const dim3 grid((max_rows + t.qt - 1) / t.qt, batch);
      const int e = wide ? launch_prompt_tc(p, pages, grid, t, stream) : static_cast<int>(launch_prompt(p, grid, t, stream));
      eredu_count_launches(1);
      return e;
    }
  }
  const TalkPlan t = talk_plan(H, G, dk, dv, max_rows, decode);
  if (t.qt == 0) return -1;
  p.qt = t.qt;
  p.octets = t.octets;
  p.warps = t.warps;
  p.lanes = t.lanes;
  p.splits = decode ? splits : 1;
  p.group_bytes = t.group_bytes;
  const dim3 grid((max_rows + t.qt - 1) / t.qt * p.splits, batch);
  const int threads = t.warps * t.lanes * 32;
  const bool small = dk <= 64 && dv <= 64;
  cudaError_t e;
  if (small && t.per_warp == 4) e = launch_talking<4, 4, 4>(p, grid, threads, t.smem, stream);
  else if (small && t.per_warp == 2) e = launch_talking<4, 4, 2>(p, grid, threads, t.smem, stream);
  else if (small) e = launch_talking<4, 4, 1>(p, grid, threads, t.smem, stream);
  else if (t.per_warp == 2) e = launch_talking<8, 8, 2>(p, grid, threads, t.smem, stream);
  else e = launch_talking<8, 8, 1>(p, grid, threads, t.smem, stream);
  eredu_count_launches(1);
  return static_cast<int>(e);
}

// The same for fp32 (fp32 = 1) or bf16 and any sizes whose query and output rows fit shared memory.
extern "C" int eredu_talking_attention_simt(const void* q, const void* k_cache, const void* v_cache, void* out, const int* block_table,
                                            const int* seq_lens, const int* cu_q, const void* talk, const float* sinks, int batch,
                                            int q_per_seq, int max_rows, int max_pages, int H, int G, int dk, int dv, int window, int keep,
                                            int fp32, float scale, float softcap, cudaStream_t stream) {
  if (batch <= 0 || max_rows <= 0) return 0;
  if (G <= 0 || H % G != 0 || dk <= 0 || dv <= 0 || window < 0 || keep < 0 || batch > 65535) return -1;
  const TalkParams p = talk_params(q, k_cache, v_cache, out, block_table, seq_lens, cu_q, talk, sinks, q_per_seq, max_pages, H, G, dk, dv,
                                   window, keep, scale, softcap);
  const size_t smem = (static_cast<size_t>(H) * (dk + dv) + kKeys * (H + 1) + H * (kKeys + 1) + 3 * H) * sizeof(float);
  if (smem > kSmemLimit - 1024) return -1;
  auto run = [&](auto kernel, bool& configured) -> cudaError_t {
    if (!configured) {
      const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemLimit - 1024);
      if (e != cudaSuccess) return e;
      configured = true;
    }
    return launch_pdl(kernel, dim3(max_rows, batch), dim3(256), smem, stream, p);
  };
  static bool done[2] = {};
  const cudaError_t e = fp32 ? run(talking_simt_kernel<float>, done[0]) : run(talking_simt_kernel<__nv_bfloat16>, done[1]);
  eredu_count_launches(1);
  return static_cast<int>(e);
}
