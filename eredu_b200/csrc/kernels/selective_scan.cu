// Selective scan (Mamba): a diagonal recurrence per channel and state whose step size, input and output vectors depend on the token.
//   dt = softplus(W_dt low + b),  S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n,  y_c = sum_n S[c, n] C_n + D_c x_c,  out = y silu(z)
// params [M, rank + 2 n] = [low | B | C]; S fp32, the first c * n elements of a sequence's state. Step sizes, decays and S are fp32.
//
// A few neighbouring lanes share a channel, each with NS states in registers; a CTA takes the channels of 128 threads and stages B, C,
// step sizes and inputs of some tokens at a time in shared memory. Because a step is affine in S and its factors over a tile
// multiply to exp(A sum dt), long portions are cut into tiles that run in parallel: one launch leaves what every tile adds to a zero
// state and its summed step size, a second one chains the tiles in front of its own and replays it.
//
// Prompts in bf16 with at most 32 states a channel take a form of their own, bound by the exponentials: a thread owns a whole channel, B and
// C come as broadcasts from shared memory, states are updated in pairs (two-wide fp32 instructions), and a part of the exponentials is
// a polynomial on the FMA pipe, which the special-function unit would otherwise hold up.
#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/launch_count.h"
#include "../common/mma.cuh"
#include "../common/ptx.cuh"
#include "../common/ragged.cuh"

namespace eredu {

template <typename T>
struct ScanParams {
  const T* x;              // [M, C]
  const T* z;              // [M, ldz]
  const T* params;         // [M, ldp]
  float* dt;               // [M, C] W_dt low, or null: formed here; the form below leaves finished step sizes in the tiles of its first launch
  const T* dt_w;           // [C, rank]
  const float* dt_b;       // [C]
  const float* A;          // [C, N]
  const float* D;          // [C]
  float* state;
  T* out;                  // [M, C]
  float* maps;             // [B, tiles, N, C] what a tile adds, then [B, tiles, C] summed step sizes
  int C, N, rank, ldz, ldp, state_elems;
  int lanes, stage, tiles, tile_len;   // lanes of a channel; tokens staged at a time; tiles of the longest portion and their length
  RaggedBatch seqs;
};

constexpr int kScanThreads = 128;
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float softplus_f32(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
// exp(dt A) S + add. With fp32 activations a slow decay is applied as S + (exp(dt A) - 1) S: rounding a factor just below one would
// add up over the tokens that a state remembers. a: A, times log2(e) for bf16 activations.
template <typename T>
__device__ __forceinline__ float scan_step(float dt, float a, float S, float add) {
  if constexpr (sizeof(T) == 4) return S + fmaf(expm1f(dt * a), S, add);
  return fmaf(ex2_approx(dt * a), S, add);
}

// MAPS: only the map of the tile, from a zero state. N4: states are whole groups of four.
template <typename T, int NS, bool MAPS>
__global__ void __launch_bounds__(kScanThreads) selective_scan_kernel(ScanParams<T> p) {
  extern __shared__ float sm[];
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.z, tile = blockIdx.y;
  const RaggedSeq s = ragged_seq(p.seqs, b);
  const int t_begin = tile * p.tile_len, t_end = min(s.rows, t_begin + p.tile_len);
  if (t_begin >= t_end) return;                                            // uniform
  if (MAPS && t_end >= s.rows) return;                                     // nothing follows the last tile
  const int lanes = p.lanes, per = kScanThreads / lanes;                   // channels of the CTA
  const int c0 = blockIdx.x * per, nc = min(per, p.C - c0);
  const int width = lanes * NS;                                            // states of a channel, filled up with silent ones
  float* bs = sm;                                                          // [stage][width]
  float* cs = bs + p.stage * width;                                        // [stage][width]
  float* ds = cs + p.stage * width;                                        // [stage][per] step size
  float* xs = ds + p.stage * per;                                          // [stage][per] input
  float* ys = xs + p.stage * per;                                          // [stage][per]
  const int ch = threadIdx.x / lanes, part = threadIdx.x % lanes, n0 = part * NS;
  const bool in = ch < nc;
  const int c = c0 + (in ? ch : 0);
  float a[NS], S[NS];
  const size_t cell = static_cast<size_t>(c) * p.N + n0;
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    a[i] = n0 + i < p.N ? p.A[cell + i] * (sizeof(T) == 4 ? 1.f : kLog2e) : 0.f;
    S[i] = 0.f;
  }
  float* st = p.state + static_cast<size_t>(s.slot) * p.state_elems + cell;
  float* maps = p.maps + static_cast<size_t>(b) * p.tiles * p.C * p.N;
  float* sums = p.maps + static_cast<size_t>(p.seqs.B) * p.tiles * p.C * p.N + static_cast<size_t>(b) * p.tiles * p.C;
  if (!MAPS) {
    if (s.live)
#pragma unroll
      for (int i = 0; i < NS; ++i) S[i] = n0 + i < p.N ? st[i] : 0.f;
    for (int j = 0; j < tile; ++j) {                                       // the tiles in front
      const float dt = sums[static_cast<size_t>(j) * p.C + c];
#pragma unroll
      for (int i = 0; i < NS; ++i)
        if (n0 + i < p.N) S[i] = scan_step<T>(dt, a[i], S[i], maps[(static_cast<size_t>(j) * p.N + n0 + i) * p.C + c]);
    }
  }
  float total = 0.f;
  const float d_skip = MAPS ? 0.f : p.D[c];
  for (int t0 = t_begin; t0 < t_end; t0 += p.stage) {
    const int n = min(p.stage, t_end - t0);
    const size_t m0 = static_cast<size_t>(s.row0 + t0);
    __syncthreads();                                                       // the previous tokens are done with
    for (int i = threadIdx.x; i < n * width; i += kScanThreads) {
      const int t = i / width, k = i - t * width;
      const T* row = p.params + (m0 + t) * p.ldp + p.rank;
      bs[i] = k < p.N ? to_f32(row[k]) : 0.f;
      if (!MAPS) cs[i] = k < p.N ? to_f32(row[p.N + k]) : 0.f;
    }
    if (p.dt != nullptr) {
      for (int i = threadIdx.x; i < n * per; i += kScanThreads) {
        const int t = i / per, k = i - t * per;
        if (k >= nc) continue;
        ds[i] = softplus_f32(p.dt[(m0 + t) * p.C + c0 + k] + p.dt_b[c0 + k]);
        xs[i] = to_f32(p.x[(m0 + t) * p.C + c0 + k]);
      }
    } else {                                                               // the lanes of a channel share its row of W_dt
      const T* w = p.dt_w + static_cast<size_t>(c) * p.rank;
      for (int t = 0; t < n; ++t) {
        const T* low = p.params + (m0 + t) * p.ldp;
        float v = 0.f;
        if constexpr (sizeof(T) == 2) {
          if ((p.rank & 7) == 0 && (p.ldp & 7) == 0) {                     // 16-byte pieces
            for (int j = part * 8; j < p.rank; j += lanes * 8) {
              const float4 w0 = load4(w + j), w1 = load4(w + j + 4), l0 = load4(low + j), l1 = load4(low + j + 4);
              v = fmaf(w0.x, l0.x, fmaf(w0.y, l0.y, fmaf(w0.z, l0.z, fmaf(w0.w, l0.w, v))));
              v = fmaf(w1.x, l1.x, fmaf(w1.y, l1.y, fmaf(w1.z, l1.z, fmaf(w1.w, l1.w, v))));
            }
          } else {
            for (int j = part; j < p.rank; j += lanes) v = fmaf(to_f32(w[j]), to_f32(low[j]), v);
          }
        } else {
          for (int j = part; j < p.rank; j += lanes) v = fmaf(to_f32(w[j]), to_f32(low[j]), v);
        }
        for (int o = lanes >> 1; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
        if (in && part == 0) {
          ds[t * per + ch] = softplus_f32(v + p.dt_b[c]);
          xs[t * per + ch] = to_f32(p.x[(m0 + t) * p.C + c]);
        }
      }
    }
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      const float dt = in ? ds[t * per + ch] : 0.f, xv = in ? xs[t * per + ch] : 0.f;
      const float dx = dt * xv;
      float y = 0.f;
#pragma unroll
      for (int i = 0; i < NS; ++i) {
        S[i] = scan_step<T>(dt, a[i], S[i], dx * bs[t * width + n0 + i]);
        if (!MAPS) y = fmaf(S[i], cs[t * width + n0 + i], y);
      }
      if (MAPS) {
        total += dt;
      } else {
        for (int o = lanes >> 1; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
        if (in && part == 0) ys[t * per + ch] = fmaf(d_skip, xv, y);
      }
    }
    if (!MAPS) {
      __syncthreads();
      for (int i = threadIdx.x; i < n * per; i += kScanThreads) {
        const int t = i / per, k = i - t * per;
        if (k >= nc) continue;
        const float g = to_f32(p.z[(m0 + t) * p.ldz + c0 + k]);
        p.out[(m0 + t) * p.C + c0 + k] = from_f32<T>(ys[i] * (sizeof(T) == 4 ? silu_f32(g) : silu_fast(g)));
      }
    }
  }
  if (!in) return;
  if (MAPS) {
#pragma unroll
    for (int i = 0; i < NS; ++i)
      if (n0 + i < p.N) maps[(static_cast<size_t>(tile) * p.N + n0 + i) * p.C + c] = S[i];
    if (part == 0) sums[static_cast<size_t>(tile) * p.C + c] = total;
  } else if (s.live && t_end >= s.rows) {
#pragma unroll
    for (int i = 0; i < NS; ++i)
      if (n0 + i < p.N) st[i] = S[i];
  }
}

// ---------------------------------------------------------------- prompts in bf16, NP pairs of states
__device__ __forceinline__ uint64_t mul_f32x2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
// 2^x for a pair, x <= 0, on the FMA pipe: n = round(x) by the 1.5 * 2^23 trick, the Taylor series of 2^f = e^(f ln 2) on f = x - n in
// [-1/2, 1/2] up to f^6 (relative error below 2e-7; exact at 0, so slow decays keep their accuracy), n added into the exponent.
__device__ __forceinline__ uint64_t ex2_pair_poly(uint64_t x) {
  float x0, x1;
  unpack_f32x2(x, x0, x1);
  x = pack_f32x2(fmaxf(x0, -126.f), fmaxf(x1, -126.f));
  const uint64_t magic = pack_f32x2(12582912.f, 12582912.f), back = pack_f32x2(-12582912.f, -12582912.f), minus = pack_f32x2(-1.f, -1.f);
  const uint64_t t = add_f32x2(x, magic);
  const uint64_t f = fma_f32x2(add_f32x2(t, back), minus, x);
  auto two = [](float c) { return pack_f32x2(c, c); };
  uint64_t y = fma_f32x2(f, two(1.5403530e-4f), two(1.3333558e-3f));      // ln(2)^k / k!
  y = fma_f32x2(y, f, two(9.6181291e-3f));
  y = fma_f32x2(y, f, two(5.5504109e-2f));
  y = fma_f32x2(y, f, two(2.4022651e-1f));
  y = fma_f32x2(y, f, two(6.9314718e-1f));
  y = fma_f32x2(y, f, two(1.f));
  float y0, y1, t0, t1;
  unpack_f32x2(y, y0, y1);
  unpack_f32x2(t, t0, t1);
  return pack_f32x2(__int_as_float(__float_as_int(y0) + (__float_as_int(t0) << 23)), __int_as_float(__float_as_int(y1) + (__float_as_int(t1) << 23)));
}
__device__ __forceinline__ uint64_t ex2_pair(uint64_t x, bool poly) {
  if (poly) return ex2_pair_poly(x);
  float a, b;
  unpack_f32x2(x, a, b);
  return pack_f32x2(ex2_approx(a), ex2_approx(b));
}
// softplus with 32-bit accuracy from the fast logarithm: log(1 + t) keeps its relative accuracy for small t by the correction
// t / ((1 + t) - 1) (Goldberg, "What every computer scientist should know about floating-point arithmetic").
__device__ __forceinline__ float softplus_fast(float x) {
  const float t = ex2_approx(-fabsf(x) * kLog2e), u = 1.f + t;
  return fmaxf(x, 0.f) + (u == 1.f ? t : __logf(u) * __fdividef(t, u - 1.f));
}

constexpr int kWideStage = 32;       // tokens of B and C staged at a time
constexpr bool kWidePoly = true;     // one of every eight pairs of exponentials on the FMA pipe (none, two and three measured slower)
constexpr int kWideAhead = 4;        // tokens whose channel values are in flight

template <int NP, bool MAPS>
__global__ void __launch_bounds__(kScanThreads, NP <= 8 ? 6 : 3) scan_wide_kernel(ScanParams<__nv_bfloat16> p) {
  using T = __nv_bfloat16;
  __shared__ __align__(16) float bc[2][kWideStage][2][2 * NP];             // buffer, token, B or C
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.z, tile = blockIdx.y;
  const RaggedSeq s = ragged_seq(p.seqs, b);
  const int t_begin = tile * p.tile_len, t_end = min(s.rows, t_begin + p.tile_len);
  if (t_begin >= t_end) return;                                            // uniform
  const bool last = t_end >= s.rows, split = p.tiles > 1;                  // nothing follows the last tile: its first launch only forms step sizes
  const int c = blockIdx.x * kScanThreads + threadIdx.x;
  const bool in = c < p.C;
  const int cc = in ? c : 0;
  uint64_t a[NP], S[NP];
  auto state_pair = [&](const float* src, int i) {
    return pack_f32x2(2 * i < p.N ? src[2 * i] : 0.f, 2 * i + 1 < p.N ? src[2 * i + 1] : 0.f);
  };
  const size_t cell = static_cast<size_t>(cc) * p.N;
#pragma unroll
  for (int i = 0; i < NP; ++i) {
    a[i] = mul_f32x2(state_pair(p.A + cell, i), pack_f32x2(kLog2e, kLog2e));
    S[i] = 0ull;
  }
  float* st = p.state + static_cast<size_t>(s.slot) * p.state_elems + cell;
  float* maps = p.maps + static_cast<size_t>(b) * p.tiles * p.C * p.N;
  float* sums = p.maps + static_cast<size_t>(p.seqs.B) * p.tiles * p.C * p.N + static_cast<size_t>(b) * p.tiles * p.C;
  if (!MAPS) {
    if (s.live)
#pragma unroll
      for (int i = 0; i < NP; ++i) S[i] = state_pair(st, i);
    for (int j = 0; j < tile; ++j) {                                       // the tiles in front
      const float dt = sums[static_cast<size_t>(j) * p.C + cc];
      const uint64_t d2 = pack_f32x2(dt, dt);
#pragma unroll
      for (int i = 0; i < NP; ++i) {
        const float* add = maps + (static_cast<size_t>(j) * p.N + 2 * i) * p.C + cc;
        S[i] = fma_f32x2(ex2_pair(mul_f32x2(d2, a[i]), false), S[i], pack_f32x2(2 * i < p.N ? add[0] : 0.f, 2 * i + 1 < p.N ? add[p.C] : 0.f));
      }
    }
  }
  const float bias = p.dt_b[cc], d_skip = MAPS ? 0.f : p.D[cc];
  const size_t m0 = static_cast<size_t>(s.row0);
  auto stage = [&](int t0, int buf) {                                      // B and C of some tokens, fp32, silent states zero
    const int n = min(kWideStage, t_end - t0);
    for (int i = threadIdx.x; i < n * 4 * NP; i += kScanThreads) {
      const int t = i / (4 * NP), k = i % (4 * NP), w = k / (2 * NP), j = k % (2 * NP);
      bc[buf][t][w][j] = j < p.N ? to_f32(p.params[(m0 + t0 + t) * p.ldp + p.rank + w * p.N + j]) : 0.f;
    }
  };
  float dn[kWideAhead];
  T xn[kWideAhead], zn[kWideAhead];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int u = 0; u < kWideAhead; ++u) {
      if (t0 + u >= t_end) break;
      const size_t m = m0 + t0 + u;
      dn[u] = p.dt[m * p.C + cc];
      xn[u] = p.x[m * p.C + cc];
      if (!MAPS) zn[u] = p.z[m * p.ldz + cc];
    }
  };
  float total = 0.f;
  if (MAPS && last) {
    if (in)
      for (size_t m = m0 + t_begin; m < m0 + t_end; ++m) p.dt[m * p.C + c] = softplus_fast(p.dt[m * p.C + c] + bias);
    return;
  }
  fetch(t_begin);
  stage(t_begin, 0);
  int buf = 0;
  for (int t0 = t_begin; t0 < t_end; t0 += kWideStage, buf ^= 1) {
    __syncthreads();                                                       // this buffer is filled, the other one left
    if (t0 + kWideStage < t_end) stage(t0 + kWideStage, buf ^ 1);
    const int n = min(kWideStage, t_end - t0);
    for (int q = 0; q < n; q += kWideAhead) {
      float dt[kWideAhead], x[kWideAhead], z[kWideAhead];
#pragma unroll
      for (int u = 0; u < kWideAhead; ++u) {
        dt[u] = !MAPS && split ? dn[u] : softplus_fast(dn[u] + bias);
        x[u] = to_f32(xn[u]);
        z[u] = MAPS ? 0.f : to_f32(zn[u]);
      }
      fetch(t0 + q + kWideAhead);
#pragma unroll
      for (int u = 0; u < kWideAhead; ++u) {
        if (q + u >= n) break;
        const uint64_t d2 = pack_f32x2(dt[u], dt[u]);
        const float dx = dt[u] * x[u];
        const uint64_t dx2 = pack_f32x2(dx, dx);
        const ulonglong2* bp = reinterpret_cast<const ulonglong2*>(bc[buf][q + u][0]);
        const ulonglong2* cp = reinterpret_cast<const ulonglong2*>(bc[buf][q + u][1]);
        uint64_t y2 = 0ull, y3 = 0ull;
#pragma unroll
        for (int i = 0; i < NP; i += 2) {
          const ulonglong2 bb = bp[i / 2];
          S[i] = fma_f32x2(ex2_pair(mul_f32x2(d2, a[i]), false), S[i], mul_f32x2(dx2, bb.x));
          S[i + 1] = fma_f32x2(ex2_pair(mul_f32x2(d2, a[i + 1]), i % 8 == 0 && kWidePoly), S[i + 1], mul_f32x2(dx2, bb.y));
          if (!MAPS) {
            const ulonglong2 cv = cp[i / 2];
            y2 = fma_f32x2(S[i], cv.x, y2);
            y3 = fma_f32x2(S[i + 1], cv.y, y3);
          }
        }
        if (MAPS) {
          total += dt[u];
          if (in) p.dt[(m0 + t0 + q + u) * p.C + c] = dt[u];
        } else if (in) {
          float y0, y1;
          unpack_f32x2(add_f32x2(y2, y3), y0, y1);
          p.out[(m0 + t0 + q + u) * p.C + c] = __float2bfloat16(fmaf(d_skip, x[u], y0 + y1) * silu_fast(z[u]));
        }
      }
    }
  }
  if (!in) return;
  if (MAPS) sums[static_cast<size_t>(tile) * p.C + c] = total;
  if (MAPS || (s.live && last)) {
    float* dst = MAPS ? maps + static_cast<size_t>(tile) * p.N * p.C + c : st;
    const size_t step = MAPS ? p.C : 1;
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      float s0, s1;
      unpack_f32x2(S[i], s0, s1);
      if (2 * i < p.N) dst[2 * i * step] = s0;
      if (2 * i + 1 < p.N) dst[(2 * i + 1) * step] = s1;
    }
  }
}

// ---------------------------------------------------------------- decode steps in bf16
// One token per sequence. A CTA takes 512 / N channels of up to eight sequences: the step sizes of all of them are one small product on the
// tensor cores, so W_dt is read once for them, and a thread then updates four states of one channel for every sequence, all its states in flight.
constexpr int kDecodeSeqs = 8;

__global__ void __launch_bounds__(kScanThreads) scan_decode_kernel(ScanParams<__nv_bfloat16> p) {
  using T = __nv_bfloat16;
  __shared__ float ds[kDecodeSeqs][64], xs[kDecodeSeqs][64], zs[kDecodeSeqs][64];
  __shared__ __align__(16) float bc[kDecodeSeqs][128];                     // B, then C
  __shared__ int slot_of[kDecodeSeqs], live[kDecodeSeqs];
  pdl_launch_early();
  const int quads = p.N / 4, per = kScanThreads / quads;                   // lanes of a channel, channels of the CTA
  const int c0 = blockIdx.x * per, b0 = blockIdx.y * kDecodeSeqs, nb = min(kDecodeSeqs, p.seqs.B - b0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tig = lane & 3;
  const int ch = threadIdx.x / quads, quad = threadIdx.x % quads, c = c0 + ch;
  const float4 a = load4(p.A + static_cast<size_t>(c) * p.N + quad * 4);   // weights and tables: nothing in front of this launch writes them
  const float bias = p.dt_b[c], d_skip = p.D[c];
  if (threadIdx.x < kDecodeSeqs)
    slot_of[threadIdx.x] = threadIdx.x < nb ? p.seqs.page_to_slot[p.seqs.block_table[static_cast<size_t>(b0 + threadIdx.x) * p.seqs.max_pages]] : 0;
  __syncthreads();
  if (threadIdx.x < nb)                                                    // the states of these channels start towards L2
    bulk_prefetch_l2(p.state + static_cast<size_t>(slot_of[threadIdx.x]) * p.state_elems + static_cast<size_t>(c0) * p.N, per * p.N * sizeof(float));
  pdl_wait();
  pdl_launch_dependents();
  if (threadIdx.x < kDecodeSeqs) live[threadIdx.x] = threadIdx.x < nb && p.seqs.slots[b0 + threadIdx.x] >= 0;
  for (int i = threadIdx.x; i < nb * per; i += kScanThreads) {
    const int q = i / per, k = i - q * per;
    const size_t m = b0 + q;
    xs[q][k] = to_f32(p.x[m * p.C + c0 + k]);
    zs[q][k] = to_f32(p.z[m * p.ldz + c0 + k]);
  }
  for (int i = threadIdx.x; i < nb * 2 * p.N; i += kScanThreads) {
    const int q = i / (2 * p.N), k = i - q * 2 * p.N;
    bc[q][k] = to_f32(p.params[static_cast<size_t>(b0 + q) * p.ldp + p.rank + k]);
  }
  // step sizes: rows are sequences (the upper eight of the product stay empty), a tile of eight channels per turn
  for (int nt = warp; nt < per / 8; nt += kScanThreads / 32) {
    const T* w = p.dt_w + static_cast<size_t>(c0 + nt * 8 + g) * p.rank + tig * 2;
    const T* low = p.params + static_cast<size_t>(b0 + min(g, nb - 1)) * p.ldp + tig * 2;
    float acc[2][4] = {};
    auto ld = [](const T* q, bool in) { return in ? *reinterpret_cast<const uint32_t*>(q) : 0u; };
#pragma unroll 8
    for (int k = 0; k < p.rank; k += 16) {
      const bool full = k + 8 < p.rank;                                    // rank is a multiple of eight
      mma16816(acc[(k >> 4) & 1], ld(low + k, true), 0u, ld(low + k + 8, full), 0u, ld(w + k, true), ld(w + k + 8, full));
    }
    ds[g][nt * 8 + tig * 2] = acc[0][0] + acc[1][0];
    ds[g][nt * 8 + tig * 2 + 1] = acc[0][1] + acc[1][1];
  }
  __syncthreads();
  float4 S[kDecodeSeqs];
  float* st = p.state + static_cast<size_t>(c) * p.N + quad * 4;
#pragma unroll
  for (int i = 0; i < kDecodeSeqs; ++i)
    if (i < nb) S[i] = load4(st + static_cast<size_t>(slot_of[i]) * p.state_elems);
#pragma unroll
  for (int i = 0; i < kDecodeSeqs; ++i) {
    if (i < nb && live[i]) {                                               // uniform
      const float dt = softplus_fast(ds[i][ch] + bias), x = xs[i][ch], dx = dt * x, d2 = dt * kLog2e;
      const float4 bv = load4(&bc[i][quad * 4]), cv = load4(&bc[i][p.N + quad * 4]);
      S[i] = make_float4(fmaf(ex2_approx(d2 * a.x), S[i].x, dx * bv.x), fmaf(ex2_approx(d2 * a.y), S[i].y, dx * bv.y),
                         fmaf(ex2_approx(d2 * a.z), S[i].z, dx * bv.z), fmaf(ex2_approx(d2 * a.w), S[i].w, dx * bv.w));
      store4(st + static_cast<size_t>(slot_of[i]) * p.state_elems, S[i]);
      float y = fmaf(S[i].x, cv.x, fmaf(S[i].y, cv.y, fmaf(S[i].z, cv.z, S[i].w * cv.w)));
      for (int o = quads >> 1; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
      if (quad == 0) p.out[static_cast<size_t>(b0 + i) * p.C + c] = __float2bfloat16(fmaf(d_skip, x, y) * silu_fast(zs[i][ch]));
    }
  }
}

static bool scan_decode_ok(const ScanParams<__nv_bfloat16>& p) {
  const int quads = p.N / 4;
  return p.seqs.cu_q == nullptr && p.seqs.q_per_seq == 1 && p.dt == nullptr && p.N >= 8 && p.N <= 64 && (p.N & (p.N - 1)) == 0 &&
         p.C % (kScanThreads / quads) == 0 && p.rank % 8 == 0 && p.ldp % 2 == 0 && p.state_elems % 4 == 0;
}

struct ScanShape {
  bool wide;
  int ns, lanes, stage, tiles, tile_len, channels;
};

static size_t scan_smem(const ScanShape& s) {
  return (static_cast<size_t>(2) * s.stage * s.lanes * s.ns + 3 * static_cast<size_t>(s.stage) * s.channels) * sizeof(float);
}

constexpr int kScanMinTile = 64;     // tokens of a tile at least

constexpr int kWideMinRows = 16;     // portions from here on take the form of a thread per channel

static ScanShape scan_shape(int C, int N, int batch, int max_rows, int sm_count, bool tiled, bool wide_ok) {
  ScanShape s;
  s.wide = wide_ok && N <= 32 && max_rows >= kWideMinRows;
  s.ns = N <= 128 ? 4 : N <= 256 ? 8 : 16;
  s.lanes = 1;
  while (s.lanes * s.ns < N) s.lanes *= 2;
  s.channels = kScanThreads / s.lanes;
  s.stage = s.lanes * s.ns <= 64 ? 32 : 8;
  while (scan_smem(s) > 48 * 1024) s.stage /= 2;
  if (s.stage > max_rows) s.stage = max_rows;
  // enough CTAs to fill the machine, in tiles of equal length
  const int per = s.wide ? kScanThreads : s.channels;
  const long long ctas = static_cast<long long>((C + per - 1) / per) * batch;
  const long long want = tiled ? (12LL * (sm_count > 0 ? sm_count : 148)) / ctas : 1;
  const int most = max_rows / kScanMinTile;
  s.tiles = static_cast<int>(want < most ? want : most);
  if (s.tiles < 1) s.tiles = 1;
  s.tile_len = (max_rows + s.tiles - 1) / s.tiles;
  s.tile_len = (s.tile_len + 31) & ~31;
  s.tiles = (max_rows + s.tile_len - 1) / s.tile_len;
  return s;
}

template <typename T, int NS>
static cudaError_t launch_scan(const ScanParams<T>& p, const ScanShape& s, cudaStream_t stream) {
  const size_t smem = scan_smem(s);
  const dim3 grid((p.C + s.channels - 1) / s.channels, s.tiles, p.seqs.B);
  if (grid.y > 65535 || grid.z > 65535) return cudaErrorInvalidValue;
  if (s.tiles > 1) {
    const cudaError_t e = launch_pdl(selective_scan_kernel<T, NS, true>, grid, dim3(kScanThreads), smem, stream, p);
    if (e != cudaSuccess) return e;
    eredu_count_launches(1);
  }
  return launch_pdl(selective_scan_kernel<T, NS, false>, grid, dim3(kScanThreads), smem, stream, p);
}

template <int NP>
static cudaError_t launch_scan_wide(const ScanParams<__nv_bfloat16>& p, const ScanShape& s, cudaStream_t stream) {
  const dim3 grid((p.C + kScanThreads - 1) / kScanThreads, s.tiles, p.seqs.B);
  if (grid.y > 65535 || grid.z > 65535) return cudaErrorInvalidValue;
  if (s.tiles > 1) {
    const cudaError_t e = launch_pdl(scan_wide_kernel<NP, true>, grid, dim3(kScanThreads), 0, stream, p);
    if (e != cudaSuccess) return e;
    eredu_count_launches(1);
  }
  return launch_pdl(scan_wide_kernel<NP, false>, grid, dim3(kScanThreads), 0, stream, p);
}

template <typename T>
static cudaError_t run_scan(const void* x, const void* z, const void* params, float* dt, const void* dt_w, const float* dt_b, const float* A,
                            const float* D, float* state, void* out, float* scratch, const ScanShape& s, int C, int N, int rank, int ldz, int ldp,
                            int state_elems, const RaggedBatch& r, cudaStream_t stream) {
  const ScanParams<T> p = {static_cast<const T*>(x), static_cast<const T*>(z), static_cast<const T*>(params), dt, static_cast<const T*>(dt_w), dt_b, A, D,
                           state, static_cast<T*>(out), scratch, C, N, rank, ldz, ldp, state_elems, s.lanes, s.stage, s.tiles, s.tile_len, r};
  if constexpr (sizeof(T) == 2) {
    if (scan_decode_ok(p)) {
      const int per = kScanThreads / (N / 4);
      return launch_pdl(scan_decode_kernel, dim3(C / per, (r.B + kDecodeSeqs - 1) / kDecodeSeqs), dim3(kScanThreads), 0, stream, p);
    }
    if (s.wide) return N <= 8 ? launch_scan_wide<4>(p, s, stream) : N <= 16 ? launch_scan_wide<8>(p, s, stream) : launch_scan_wide<16>(p, s, stream);
  }
  return s.ns == 4 ? launch_scan<T, 4>(p, s, stream) : s.ns == 8 ? launch_scan<T, 8>(p, s, stream) : launch_scan<T, 16>(p, s, stream);
}

}  // namespace eredu

using namespace eredu;

// fp32 elements of scratch that let a call over `rows` rows of `batch` sequences run its tiles in parallel (0: one tile each).
extern "C" long long eredu_selective_scan_scratch_elems(int channels, int states, int batch, int max_rows, int sm_count, int fp32) {
  const ScanShape s = scan_shape(channels, states, batch, max_rows, sm_count, true, fp32 == 0);
  return s.tiles > 1 ? static_cast<long long>(batch) * s.tiles * channels * (states + 1LL) : 0;
}

// dt: fp32 [M, channels] = dt_w low (overwritten), or null (formed in the kernel); scratch: fp32 [eredu_selective_scan_scratch_elems(...)] or null.
// At most 512 states a channel.
extern "C" int eredu_selective_scan(const void* x, const void* z, const void* params, float* dt, const void* dt_w, const float* dt_b,
                                    const float* A, const float* D, float* state, void* out, float* scratch, const int* block_table,
                                    const int* page_to_slot, const int* cu_q, const long long* slots, int channels, int states, int rank, int ldz,
                                    int ldp, int state_elems, int batch, int q_per_seq, int max_rows, int max_pages, int fp32, int sm_count,
                                    cudaStream_t stream) {
  if (batch <= 0 || max_rows <= 0) return 0;
  if (channels <= 0 || states <= 0 || states > 512 || rank <= 0) return -1;
  const RaggedBatch r = {block_table, page_to_slot, cu_q, slots, batch, q_per_seq, max_pages};
  const ScanShape s = scan_shape(channels, states, batch, max_rows, sm_count, scratch != nullptr, fp32 == 0 && dt != nullptr);
  const cudaError_t e = fp32 ? run_scan<float>(x, z, params, dt, dt_w, dt_b, A, D, state, out, scratch, s, channels, states, rank, ldz, ldp, state_elems, r, stream)
                             : run_scan<__nv_bfloat16>(x, z, params, dt, dt_w, dt_b, A, D, state, out, scratch, s, channels, states, rank, ldz, ldp,
                                                       state_elems, r, stream);
  eredu_count_launches(1);
  return static_cast<int>(e);
}
