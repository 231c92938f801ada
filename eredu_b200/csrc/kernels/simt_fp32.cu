// CUDA-core kernels in true 32-bit arithmetic: the linear layer and paged attention of models that run in fp32, and of bf16
// shapes the tensor-core kernels do not take (row pitches a TMA descriptor cannot express, head sizes beyond 128 or not a
// multiple of 8).
#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/launch_count.h"
#include "../common/pooled.cuh"
#include "../common/ptx.cuh"

namespace eredu {

constexpr int kTile = 64, kTileK = 16;

// Y[M, N] = act(X[M, K] W[N, K]^T + bias): 64 x 64 outputs per CTA, 4 x 4 per thread, K in steps of 16 through shared memory.
// GATED: W holds N gate rows, then N up rows, Y = act(gate) * up.
template <typename T, typename TO, bool GATED>
__global__ void __launch_bounds__(256) gemm_simt_kernel(const T* __restrict__ x, const T* __restrict__ w, TO* __restrict__ y,
                                                         const T* __restrict__ bias, int M, int N, int K, int ldx, int ldw, int ldy,
                                                         int act, float act_a, float act_b) {
  constexpr int PARTS = GATED ? 2 : 1;
  __shared__ float xs[kTileK][kTile + 4], ws[PARTS][kTileK][kTile + 4];
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int n0 = blockIdx.x * kTile, m0 = blockIdx.y * kTile;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[PARTS][4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kTileK) {
    for (int i = threadIdx.x; i < kTile * kTileK; i += 256) {
      const int r = i / kTileK, k = i % kTileK;
      xs[k][r] = (m0 + r < M && k0 + k < K) ? to_f32(x[static_cast<size_t>(m0 + r) * ldx + k0 + k]) : 0.f;
#pragma unroll
      for (int d = 0; d < PARTS; ++d)
        ws[d][k][r] = (n0 + r < N && k0 + k < K) ? to_f32(w[static_cast<size_t>(d * N + n0 + r) * ldw + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kTileK; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&xs[k][ty * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
      for (int d = 0; d < PARTS; ++d) {
        const float4 b = *reinterpret_cast<const float4*>(&ws[d][k][tx * 4]);
        const float bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[d][i][j] = fmaf(av[i], bv[j], acc[d][i][j]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) break;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= N) break;
      float v = acc[0][i][j] + (bias != nullptr ? to_f32(bias[n]) : 0.f);
      if (GATED) {
        v = act == 3 ? fmaxf(v, 0.f) : silu_f32(v);
        v *= acc[PARTS - 1][i][j] + (bias != nullptr ? to_f32(bias[N + n]) : 0.f);
      } else if (act == 1) {
        v = fmaxf(v, 0.f);
        v *= v;
      } else if (act == 4) {
        v = xielu<false>(v, act_a, act_b);
      }
      y[static_cast<size_t>(m) * ldy + n] = from_f32<TO>(v);
    }
  }
}

// Expert GEMMs over the work items of a routing plan ({expert, first row, rows, -}): Y[row] = X[index ? index[row] : row] W_e^T, or
// with DUAL silu(X Wg^T) * (X Wu^T), Wg / Wu the first / following N rows of the expert's matrix. A CTA takes 64 rows at most.
template <typename T, bool DUAL>
__global__ void __launch_bounds__(256) gemm_simt_grouped_kernel(const T* __restrict__ x, const T* __restrict__ w, T* __restrict__ y,
                                                                 const int4* __restrict__ work, const int* __restrict__ index, int N,
                                                                 int K, int ldx, int ldy, int w_rows) {
  __shared__ float xs[kTileK][kTile + 4], ws[DUAL ? 2 : 1][kTileK][kTile + 4];
  __shared__ int src[kTile];
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int4 item = work[blockIdx.y];
  const int rows = min(item.z, kTile);
  if (rows <= 0) return;
  const int n0 = blockIdx.x * kTile;
  const T* we = w + static_cast<size_t>(item.x) * w_rows * K;
  if (threadIdx.x < kTile) src[threadIdx.x] = threadIdx.x < rows ? (index != nullptr ? index[item.y + threadIdx.x] : item.y + threadIdx.x) : 0;
  __syncthreads();
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[DUAL ? 2 : 1][4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kTileK) {
    for (int i = threadIdx.x; i < kTile * kTileK; i += 256) {
      const int r = i / kTileK, k = i % kTileK;
      const bool kin = k0 + k < K, nin = kin && n0 + r < N;
      xs[k][r] = r < rows && kin ? to_f32(x[static_cast<size_t>(src[r]) * ldx + k0 + k]) : 0.f;
      ws[0][k][r] = nin ? to_f32(we[static_cast<size_t>(n0 + r) * K + k0 + k]) : 0.f;
      if constexpr (DUAL) ws[1][k][r] = nin ? to_f32(we[static_cast<size_t>(N + n0 + r) * K + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kTileK; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&xs[k][ty * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
      for (int d = 0; d < (DUAL ? 2 : 1); ++d) {
        const float4 b = *reinterpret_cast<const float4*>(&ws[d][k][tx * 4]);
        const float bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[d][i][j] = fmaf(av[i], bv[j], acc[d][i][j]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = ty * 4 + i;
    if (r >= rows) break;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= N) break;
      y[static_cast<size_t>(item.y + r) * ldy + n] = from_f32<T>(DUAL ? silu_f32(acc[0][i][j]) * acc[DUAL ? 1 : 0][i][j] : acc[0][i][j]);
    }
  }
}

struct AttnSimtParams {
  const void* q;         // [total_q, n_q, dk]
  const void* k_cache;   // [pages, n_kv, 16, dk]
  const void* v_cache;   // [pages, n_kv, 16, ldv], of which the first dv entries of a row are the value
  void* out;             // [total_q, n_q, dv]
  const int* block_table;
  const int* seq_lens;
  const int* cu_q;       // null: q_per_seq queries per sequence
  const float* sinks;    // [n_q] or null
  int q_per_seq, max_pages, n_q, n_kv, dk, dv, ldv, window, chunk;
  float scale;
  // pool > 0: the mean key and value of every block of `pool` tokens that ends before the window is seen as well
  const void* pk;        // [pages, n_kv, pool_rows, dk], page of the block's last token
  const void* pv;        // [pages, n_kv, pool_rows, dv]
  int pool, pool_rows;
};

constexpr int kMaxValueRegs = 32;  // value widths up to 1024

// One CTA per (query token, head); its four warps take every fourth group of 32 keys, one key per lane for the scores and
// one value column per lane for the sum, each with a running maximum of its own; merged at the end.
template <typename T>
__global__ void __launch_bounds__(128) attn_simt_kernel(AttnSimtParams p) {
  extern __shared__ float sm[];
  float* qs = sm;                      // [dk]
  float* merge = sm + p.dk;            // [4][dv + 2]
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.z, h = blockIdx.y, qi = blockIdx.x;
  const int q0 = p.cu_q != nullptr ? p.cu_q[b] : b * p.q_per_seq;
  const int q_len = p.cu_q != nullptr ? p.cu_q[b + 1] - q0 : p.q_per_seq;
  if (qi >= q_len) return;
  const int pos = p.seq_lens[b] - q_len + qi;
  const int kvh = h / (p.n_q / p.n_kv);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int* bt = p.block_table + static_cast<size_t>(b) * p.max_pages;
  const T* q = static_cast<const T*>(p.q) + (static_cast<size_t>(q0 + qi) * p.n_q + h) * p.dk;
  for (int i = threadIdx.x; i < p.dk; i += 128) qs[i] = to_f32(q[i]) * p.scale;
  __syncthreads();
  int lo = 0;
  if (p.window > 0) lo = max(0, pos - p.window + 1);
  else if (p.chunk > 0) lo = pos - pos % p.chunk;
  float acc[kMaxValueRegs];
#pragma unroll
  for (int c = 0; c < kMaxValueRegs; ++c) acc[c] = 0.f;
  float m = -INFINITY, l = 0.f;
  // one group of up to 32 keys: `row` names the lane's row of `keys` and `values` where it has one
  auto group = [&](const T* keys, const T* values, size_t row, bool ok, int n) {
    float s = -INFINITY;
    if (ok) {
      const T* k = keys + row * p.dk;
      s = 0.f;
      for (int i = 0; i < p.dk; ++i) s = fmaf(qs[i], to_f32(k[i]), s);
    }
    float mx = s;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    const float m_new = fmaxf(m, mx);
    const float corr = expf(m - m_new);
    const float pe = ok ? expf(s - m_new) : 0.f;
    m = m_new;
    l = l * corr + warp_sum_f32(pe);
#pragma unroll
    for (int c = 0; c < kMaxValueRegs; ++c) acc[c] *= corr;
    for (int j = 0; j < n; ++j) {
      const float pj = __shfl_sync(0xffffffffu, pe, j);
      const size_t rj = __shfl_sync(0xffffffffu, static_cast<unsigned long long>(row), j);
      const T* v = values + rj * p.ldv;
#pragma unroll
      for (int c = 0; c < kMaxValueRegs; ++c)
        if (lane + 32 * c < p.dv) acc[c] = fmaf(pj, to_f32(v[lane + 32 * c]), acc[c]);
    }
  };
  if (p.pool > 0) {
    const int blocks = pooled_seen(pos, p.window, p.pool);
    for (int b0 = warp * 32; b0 < blocks; b0 += 128) {
      const int blk = b0 + lane;
      const bool ok = blk < blocks;
      const PooledRow r = pooled_row(ok ? blk : 0, p.pool);
      const size_t row = (static_cast<size_t>(bt[r.page]) * p.n_kv + kvh) * p.pool_rows + r.row;
      group(static_cast<const T*>(p.pk), static_cast<const T*>(p.pv), row, ok, min(32, blocks - b0));
    }
  }
  for (int k0 = lo + warp * 32; k0 <= pos; k0 += 128) {
    const int key = k0 + lane;
    const bool ok = key <= pos;
    const size_t row = ok ? (static_cast<size_t>(bt[key >> 4]) * p.n_kv + kvh) * 16 + (key & 15) : 0;
    group(static_cast<const T*>(p.k_cache), static_cast<const T*>(p.v_cache), row, ok, min(32, pos - k0 + 1));
  }
  float* mine = merge + warp * (p.dv + 2);
#pragma unroll
  for (int c = 0; c < kMaxValueRegs; ++c)
    if (lane + 32 * c < p.dv) mine[lane + 32 * c] = acc[c];
  if (lane == 0) {
    mine[p.dv] = m;
    mine[p.dv + 1] = l;
  }
  __syncthreads();
  float M = p.sinks != nullptr ? p.sinks[h] : -INFINITY;
  for (int w = 0; w < 4; ++w) M = fmaxf(M, merge[w * (p.dv + 2) + p.dv]);
  float L = p.sinks != nullptr ? expf(p.sinks[h] - M) : 0.f, e[4];
  for (int w = 0; w < 4; ++w) {
    e[w] = expf(merge[w * (p.dv + 2) + p.dv] - M);
    L += merge[w * (p.dv + 2) + p.dv + 1] * e[w];
  }
  T* out = static_cast<T*>(p.out) + (static_cast<size_t>(q0 + qi) * p.n_q + h) * p.dv;
  for (int d = threadIdx.x; d < p.dv; d += 128) {
    float o = 0.f;
    for (int w = 0; w < 4; ++w) o += merge[w * (p.dv + 2) + d] * e[w];
    out[d] = from_f32<T>(o / L);
  }
}

}  // namespace eredu

using namespace eredu;

// X [M, K], W [N, K], bias [N] (or null) fp32 (in_fp32 = 1) or bf16; Y [M, N] fp32 or bf16. act 1: squared ReLU; act 4: xIELU
// with factors act_a and act_b; act 2, 3: W is [2 N, K], Y = silu(gate) * up or relu(gate) * up (bias [2 N]).
extern "C" int eredu_gemm_simt(const void* x, const void* w, void* y, const void* bias, int M, int N, int K, int ldx, int ldw, int ldy,
                               int in_fp32, int out_fp32, int act, float act_a, float act_b, cudaStream_t stream) {
  if (M <= 0 || N <= 0 || K <= 0) return 0;
  const bool gated = act == 2 || act == 3;
  const dim3 grid((N + kTile - 1) / kTile, (M + kTile - 1) / kTile);
  if (grid.y > 65535 || (in_fp32 && !out_fp32)) return -1;
  cudaError_t e;
  using B = __nv_bfloat16;
#define ER_SIMT(T_, TO_, G_)                                                                                                     \
  launch_pdl(gemm_simt_kernel<T_, TO_, G_>, grid, dim3(256), 0, stream, static_cast<const T_*>(x), static_cast<const T_*>(w),      \
             static_cast<TO_*>(y), static_cast<const T_*>(bias), M, N, K, ldx, ldw, ldy, act, act_a, act_b)
  if (in_fp32) e = gated ? ER_SIMT(float, float, true) : ER_SIMT(float, float, false);
  else if (out_fp32) e = gated ? ER_SIMT(B, float, true) : ER_SIMT(B, float, false);
  else e = gated ? ER_SIMT(B, B, true) : ER_SIMT(B, B, false);
#undef ER_SIMT
  eredu_count_launches(1);
  return static_cast<int>(e);
}

// Causal attention over the paged cache for any key width and value widths up to 1024; arguments as the tensor-core kernels. Rows of
// v_cache are ldv >= dv wide: the values may be the head of a wider row (latent attention passes the same rows as keys and values).
static int attn_simt_impl(const void* q, const void* k_cache, const void* v_cache, const void* pk, const void* pv, void* out, const int* block_table,
                               const int* seq_lens, const int* cu_q, const float* sinks, int batch, int q_per_seq, int max_q_len,
                               int max_pages, int n_q, int n_kv, int dk, int dv, int ldv, int window, int chunk, int pool, int pool_rows, int fp32, float scale,
                               cudaStream_t stream) {
  if (batch <= 0 || max_q_len <= 0) return 0;
  if (n_kv <= 0 || n_q % n_kv != 0 || dk <= 0 || dv <= 0 || dv > 32 * kMaxValueRegs || ldv < dv || window < 0 || chunk < 0) return -1;
  AttnSimtParams p;
  p.q = q;
  p.k_cache = k_cache;
  p.v_cache = v_cache;
  p.out = out;
  p.block_table = block_table;
  p.seq_lens = seq_lens;
  p.cu_q = cu_q;
  p.sinks = sinks;
  p.q_per_seq = q_per_seq;
  p.max_pages = max_pages;
  p.n_q = n_q;
  p.n_kv = n_kv;
  p.dk = dk;
  p.dv = dv;
  p.ldv = ldv;
  p.window = window;
  p.chunk = chunk;
  p.scale = scale;
  p.pk = pk;
  p.pv = pv;
  p.pool = pool;
  p.pool_rows = pool_rows;
  const size_t smem = (dk + 4 * static_cast<size_t>(dv + 2)) * sizeof(float);
  if (smem > 48 * 1024) return -1;
  const dim3 grid(max_q_len, n_q, batch);
  const cudaError_t e = fp32 ? launch_pdl(attn_simt_kernel<float>, grid, dim3(128), smem, stream, p)
                             : launch_pdl(attn_simt_kernel<__nv_bfloat16>, grid, dim3(128), smem, stream, p);
  eredu_count_launches(1);
  return static_cast<int>(e);
}

extern "C" int eredu_attn_simt(const void* q, const void* k_cache, const void* v_cache, void* out, const int* block_table,
                               const int* seq_lens, const int* cu_q, const float* sinks, int batch, int q_per_seq, int max_q_len,
                               int max_pages, int n_q, int n_kv, int dk, int dv, int ldv, int window, int chunk, int fp32, float scale,
                               cudaStream_t stream) {
  return attn_simt_impl(q, k_cache, v_cache, nullptr, nullptr, out, block_table, seq_lens, cu_q, sinks, batch, q_per_seq, max_q_len, max_pages,
                        n_q, n_kv, dk, dv, ldv, window, chunk, 0, 0, fp32, scale, stream);
}

// The same over a sliding window and the means of the blocks of `pool` tokens behind it (pk, pv as eredu_pool_blocks leaves them).
extern "C" int eredu_attn_simt_pooled(const void* q, const void* k_cache, const void* v_cache, const void* pk, const void* pv, void* out,
                                      const int* block_table, const int* seq_lens, const int* cu_q, int batch, int q_per_seq, int max_q_len,
                                      int max_pages, int n_q, int n_kv, int dk, int dv, int window, int pool, int pool_rows, int fp32,
                                      float scale, cudaStream_t stream) {
  if (window <= 0 || pool <= 0 || pool_rows <= 0 || pk == nullptr || pv == nullptr) return -1;
  return attn_simt_impl(q, k_cache, v_cache, pk, pv, out, block_table, seq_lens, cu_q, nullptr, batch, q_per_seq, max_q_len, max_pages, n_q,
                        n_kv, dk, dv, dv, window, 0, pool, pool_rows, fp32, scale, stream);
}

// work [n_work] int4 items of at most 64 rows; w [experts, w_rows, K] (dual: gate rows, then up rows); index: source row of every row of
// X (null: the row itself). X, W and Y fp32 or bf16 alike.
extern "C" int eredu_gemm_simt_grouped(const void* x, const void* w, void* y, const int* work, int n_work, const int* index, int N, int K,
                                       int ldx, int ldy, int w_rows, int dual, int fp32, cudaStream_t stream) {
  if (n_work <= 0 || N <= 0 || K <= 0) return 0;
  if (n_work > 65535) return -1;
  const dim3 grid((N + kTile - 1) / kTile, n_work);
  const int4* items = reinterpret_cast<const int4*>(work);
  cudaError_t e;
#define ER_GROUPED_SIMT(T_, D_)                                                                                                \
  e = launch_pdl(gemm_simt_grouped_kernel<T_, D_>, grid, dim3(256), 0, stream, static_cast<const T_*>(x), static_cast<const T_*>(w), \
                 static_cast<T_*>(y), items, index, N, K, ldx, ldy, w_rows)
  if (fp32 && dual) ER_GROUPED_SIMT(float, true);
  else if (fp32) ER_GROUPED_SIMT(float, false);
  else if (dual) ER_GROUPED_SIMT(__nv_bfloat16, true);
  else ER_GROUPED_SIMT(__nv_bfloat16, false);
#undef ER_GROUPED_SIMT
  eredu_count_launches(1);
  return static_cast<int>(e);
}
