// Causal depthwise convolutions over ranges of a projection's columns, and what directly follows them:
//   * heads [q | k | v]: rotation of q and k (neighbouring pairs), a factor per query head, keys and values into the paged cache
//   * channels: bias and SiLU
// y_t = sum_j taps[j] u_(t - L + 1 + j); the last L - 1 inputs of a sequence are fp32 rows of its recurrent state. Portions of
// prompts and single decoded tokens alike; bf16 or fp32 activations.
// pool_blocks: mean keys and values of blocks of cached tokens, written beside the page of a block's last token and, for the prompt
// attention, as dense rows.
#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/launch_count.h"
#include "../common/pooled.cuh"
#include "../common/ptx.cuh"
#include "../common/ragged.cuh"

namespace eredu {

struct ConvProjectParams {
  const void* proj;
  float* state;
  void* q_out;             // [M, n_q, dk]
  void* x_out;             // [M, width]
  const float* h_taps;     // [hl, heads' channels]
  const float* c_taps;     // [cl, width]
  const float* c_bias;     // [width] or null
  void* k_cache;           // [pages, n_kv, 16, dk]
  void* v_cache;           // [pages, n_kv, 16, dv]
  void* pk;                // means [pages, n_kv, pool_rows, dk]
  void* pv;
  const float* inv_freq;
  const float* q_scale;    // [n_q] or null
  const int* positions;
  const int* seq_lens;
  RaggedBatch seqs;
  int ld, state_elems, hl, cl, n_q, n_kv, dk, dv, rot, pool, pool_rows, h_hist, width, c_start, c_hist;
  int h_blocks, seg_len;   // CTAs along x that take heads; tokens of a segment
};

constexpr int kConvThreads = 128;
constexpr int kConvSeg = 16;          // tokens of a segment of a long portion
constexpr int kMaxRot = 256;          // rotated dims of a head

// VEC neighbouring elements; of a pair (VEC = 2) only the first `nv` exist.
template <typename T, int VEC>
__device__ __forceinline__ void load_vec(const T* p, float (&v)[VEC], int nv) {
  if constexpr (VEC >= 4) {
#pragma unroll
    for (int i = 0; i < VEC; i += 4) {
      const float4 a = load4(p + i);
      v[i] = a.x, v[i + 1] = a.y, v[i + 2] = a.z, v[i + 3] = a.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = i < nv ? to_f32(p[i]) : 0.f;
  }
}
template <typename T, int VEC>
__device__ __forceinline__ void store_vec(T* p, const float (&v)[VEC], int nv) {
  if constexpr (VEC >= 4) {
#pragma unroll
    for (int i = 0; i < VEC; i += 4) store4(p + i, make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]));
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i)
      if (i < nv) p[i] = from_f32<T>(v[i]);
  }
}

// VEC neighbouring elements as they lie in memory.
template <typename T, int VEC>
struct alignas(VEC == 4 ? 4 * sizeof(T) : sizeof(T)) RawVec {
  T v[VEC];
};
template <typename T, int VEC>
__device__ __forceinline__ RawVec<T, VEC> load_raw(const T* p, int nv) {
  RawVec<T, VEC> r;
  if constexpr (VEC == 4) {
    r = *reinterpret_cast<const RawVec<T, VEC>*>(p);
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) r.v[i] = i < nv ? p[i] : from_f32<T>(0.f);
  }
  return r;
}
// fp32 rows of taps and histories: whole 16-byte pieces when VEC = 4
template <int VEC>
__device__ __forceinline__ void load_row(const float* p, float (&v)[VEC], int nv) {
  load_vec<float, VEC>(p, v, nv);
}

// Walks one segment of a sequence for VEC neighbouring channels: `emit(t, y)` gets the convolved values of row t. Only the first
// segment reads the old history and writes the new one, and a segment is at least as long as the history, so no other CTA
// races it. L taps at compile time keep the window in registers and four rows in flight; L = 0: any number, rows are read again.
template <typename T, int VEC, int L, typename Emit>
__device__ __forceinline__ void conv_walk(const T* col, int ld, const float* taps, int taps_ld, int n_taps, float* hist, int nv, int n, int t0, int t1, bool live, Emit emit) {
  auto input = [&](int t, float (&v)[VEC]) {
    if (t >= 0) {
      load_vec<T, VEC>(col + static_cast<size_t>(t) * ld, v, nv);
    } else if (live) {
      load_row<VEC>(hist + static_cast<size_t>(n_taps - 1 + t) * taps_ld, v, nv);
    } else {
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = 0.f;
    }
  };
  if constexpr (L > 0) {
    constexpr int U = 4;
    float w[L][VEC], win[L - 1][VEC];
#pragma unroll
    for (int j = 0; j < L; ++j) load_row<VEC>(taps + static_cast<size_t>(j) * taps_ld, w[j], nv);
#pragma unroll
    for (int j = 0; j + 1 < L; ++j) input(t0 - (L - 1) + j, win[j]);
    for (int t = t0; t < t1; t += U) {
      RawVec<T, VEC> raw[U];
#pragma unroll
      for (int u = 0; u < U; ++u)
        if (t + u < t1) raw[u] = load_raw<T, VEC>(col + static_cast<size_t>(t + u) * ld, nv);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        if (t + u >= t1) break;
        float y[VEC];
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          const float now = to_f32(raw[u].v[i]);
          float a = w[0][i] * win[0][i];
#pragma unroll
          for (int j = 1; j + 1 < L; ++j) a = fmaf(w[j][i], win[j][i], a);
          y[i] = fmaf(w[L - 1][i], now, a);
#pragma unroll
          for (int j = 0; j + 2 < L; ++j) win[j][i] = win[j + 1][i];
          win[L - 2][i] = now;
        }
        emit(t + u, y);
      }
    }
  } else {
    for (int t = t0; t < t1; ++t) {
      float y[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) y[i] = 0.f;
      for (int j = 0; j < n_taps; ++j) {
        float v[VEC], w[VEC];
        input(t - (n_taps - 1) + j, v);
        load_row<VEC>(taps + static_cast<size_t>(j) * taps_ld, w, nv);
#pragma unroll
        for (int i = 0; i < VEC; ++i) y[i] = fmaf(w[i], v[i], y[i]);
      }
      emit(t, y);
    }
  }
  if (t0 == 0 && live)
    for (int j = 0; j + 1 < n_taps; ++j) {                  // in order: row j comes from a later row of the history or from the portion
      float v[VEC];
      input(n - (n_taps - 1) + j, v);
      store_vec<float, VEC>(hist + static_cast<size_t>(j) * taps_ld, v, nv);
    }
}

template <typename T, int VEC, typename Emit>
__device__ __forceinline__ void conv_any(const T* col, int ld, const float* taps, int taps_ld, int n_taps, float* hist, int nv, int n, int t0, int t1, bool live, Emit emit) {
  switch (n_taps) {
    case 2: return conv_walk<T, VEC, 2>(col, ld, taps, taps_ld, n_taps, hist, nv, n, t0, t1, live, emit);
    case 3: return conv_walk<T, VEC, 3>(col, ld, taps, taps_ld, n_taps, hist, nv, n, t0, t1, live, emit);
    case 4: return conv_walk<T, VEC, 4>(col, ld, taps, taps_ld, n_taps, hist, nv, n, t0, t1, live, emit);
    default: return conv_walk<T, VEC, 0>(col, ld, taps, taps_ld, n_taps, hist, nv, n, t0, t1, live, emit);
  }
}

// Mean over the rows of one block for VEC columns of one head, oldest row first.
template <typename T, int VEC>
__device__ __forceinline__ void block_mean(const T* cache, const int* bt, int n_kv, int d, int head, int col, int block, int pool, float (&m)[VEC], int nv) {
#pragma unroll
  for (int i = 0; i < VEC; ++i) m[i] = 0.f;
  for (int j = 0; j < pool; ++j) {
    const int pos = block * pool + j;
    float v[VEC];
    load_vec<T, VEC>(cache + ((static_cast<size_t>(bt[pos >> 4]) * n_kv + head) * 16 + (pos & 15)) * d + col, v, nv);
#pragma unroll
    for (int i = 0; i < VEC; ++i) m[i] += v[i];
  }
  const float n = static_cast<float>(pool);
#pragma unroll
  for (int i = 0; i < VEC; ++i) m[i] /= n;
}

// Grid (blocks of channels: heads, then channels; segments; sequences). VEC = 4: head widths and columns are whole groups of four
// channels, which a thread owns. VEC = 2: any width; a thread owns a pair of a head (or the last channel of an odd one).
template <typename T, int VEC>
__global__ void __launch_bounds__(kConvThreads, 7) conv_project_kernel(ConvProjectParams p) {
  __shared__ float cs[kConvSeg * kMaxRot / 2], sn[kConvSeg * kMaxRot / 2];
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.z;
  const RaggedSeq s = ragged_seq(p.seqs, b);
  const int t0 = blockIdx.y * p.seg_len, t1 = min(s.rows, t0 + p.seg_len);
  if (t0 >= t1) return;                                     // uniform
  const T* rows = static_cast<const T*>(p.proj) + static_cast<size_t>(s.row0) * p.ld;
  float* st = p.state + static_cast<size_t>(s.slot) * p.state_elems;
  if (static_cast<int>(blockIdx.x) >= p.h_blocks) {
    const int c = ((blockIdx.x - p.h_blocks) * kConvThreads + threadIdx.x) * VEC;
    if (c >= p.width) return;
    const int nv = min(VEC, p.width - c);
    float bias[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) bias[i] = p.c_bias != nullptr && i < nv ? p.c_bias[c + i] : 0.f;
    T* out = static_cast<T*>(p.x_out) + static_cast<size_t>(s.row0) * p.width + c;
    conv_any<T, VEC>(rows + p.c_start + c, p.ld, p.c_taps + c, p.width, p.cl, st + p.c_hist + c, nv, s.rows, t0, t1, s.live, [&](int t, float (&y)[VEC]) {
#pragma unroll
      for (int i = 0; i < VEC; ++i) y[i] = sizeof(T) == 4 ? silu_f32(y[i] + bias[i]) : silu_fast(y[i] + bias[i]);
      store_vec<T, VEC>(out + static_cast<size_t>(t) * p.width, y, nv);
    });
    return;
  }
  const int qn = p.n_q * p.dk, kn = p.n_kv * p.dk, all = qn + kn + p.n_kv * p.dv;
  const int uk = (p.dk + VEC - 1) / VEC, uv = (p.dv + VEC - 1) / VEC;      // threads of a key / value head
  const int unit0 = blockIdx.x * kConvThreads, unit = unit0 + threadIdx.x, keys = (p.n_q + p.n_kv) * uk;
  const int half = p.rot >> 1;
  if (unit0 < keys) {                                       // angles of this segment, shared by all its heads
    for (int i = threadIdx.x; i < (t1 - t0) * half; i += kConvThreads) {
      const int t = i / half, j = i - t * half;
      sincosf(static_cast<float>(p.positions[s.row0 + t0 + t]) * p.inv_freq[j], &sn[i], &cs[i]);
    }
    __syncthreads();
  }
  if (unit >= keys + p.n_kv * uv) return;
  const bool is_q = unit < p.n_q * uk, is_v = unit >= keys;
  const int rel = is_q ? unit : is_v ? unit - keys : unit - p.n_q * uk;
  const int d = is_v ? p.dv : p.dk, per = is_v ? uv : uk;
  const int head = rel / per, j = (rel - head * per) * VEC, nv = min(VEC, d - j);
  const int c = (is_q ? 0 : is_v ? qn + kn : qn) + head * d + j;
  const float scale = is_q && p.q_scale != nullptr ? p.q_scale[head] : 1.f;
  T* q = static_cast<T*>(p.q_out) + static_cast<size_t>(s.row0) * qn + c;
  T* cache = static_cast<T*>(is_v ? p.v_cache : p.k_cache);
  T* means = static_cast<T*>(is_v ? p.pv : p.pk);
  const int* bt = p.seqs.block_table + static_cast<size_t>(b) * p.seqs.max_pages;
  const int pos0 = p.pool > 0 ? p.seq_lens[b] - s.rows : 0;
  conv_any<T, VEC>(rows + c, p.ld, p.h_taps + c, all, p.hl, st + p.h_hist + c, nv, s.rows, t0, t1, s.live, [&](int t, float (&y)[VEC]) {
    if (!is_v) {
      const float* ct = cs + (t - t0) * half;
      const float* stt = sn + (t - t0) * half;
#pragma unroll
      for (int i = 0; i + 1 < VEC; i += 2)
        if (j + i < p.rot) {
          const float u = y[i], v = y[i + 1], co = ct[(j + i) >> 1], si = stt[(j + i) >> 1];
          y[i] = u * co - v * si;
          y[i + 1] = v * co + u * si;
        }
    }
    if (is_q) {
#pragma unroll
      for (int i = 0; i < VEC; ++i) y[i] *= scale;
      store_vec<T, VEC>(q + static_cast<size_t>(t) * qn, y, nv);
      return;
    }
    const long long slot = p.seqs.slots[s.row0 + t];
    if (slot < 0) return;
    store_vec<T, VEC>(cache + ((static_cast<size_t>(slot >> 4) * p.n_kv + head) * 16 + static_cast<size_t>(slot & 15)) * d + j, y, nv);
    if (p.pool > 0 && (pos0 + t + 1) % p.pool == 0) {       // this thread has written its columns of every row of the block, now or before
      const int block = (pos0 + t) / p.pool;
      const PooledRow r = pooled_row(block, p.pool);
      float m[VEC];
      block_mean<T, VEC>(cache, bt, p.n_kv, d, head, j, block, p.pool, m, nv);
      store_vec<T, VEC>(means + ((static_cast<size_t>(bt[r.page]) * p.n_kv + head) * p.pool_rows + r.row) * d + j, m, nv);
    }
  });
}

struct PoolParams {
  const void* k_cache;
  const void* v_cache;
  void* pk;
  void* pv;
  void* k_rows;            // [rows, n_kv, dk] or null
  void* v_rows;
  const int* block_table;
  const int* seq_lens;
  const int* cu_q;
  const int* first;        // [B] first dense row of a sequence
  int max_pages, n_kv, dk, dv, pool, pool_rows;
};

// Grid (blocks, sequences): one CTA per block, keys and values of all heads.
template <typename T, int VEC>
__global__ void __launch_bounds__(128) pool_blocks_kernel(PoolParams p) {
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.y, block = blockIdx.x;
  const int kv_len = p.seq_lens[b], q_len = p.cu_q[b + 1] - p.cu_q[b];
  if (q_len <= 0 || block >= kv_len / p.pool) return;
  const bool fresh = block * p.pool + p.pool > kv_len - q_len;             // completed by the new tokens
  if (!fresh && p.k_rows == nullptr) return;
  const int* bt = p.block_table + static_cast<size_t>(b) * p.max_pages;
  const PooledRow r = pooled_row(block, p.pool);
  const size_t cell = static_cast<size_t>(bt[r.page]) * p.n_kv;
  const int kq = p.n_kv * p.dk / VEC, vq = p.n_kv * p.dv / VEC;
  for (int i = threadIdx.x; i < kq + vq; i += 128) {
    const bool is_v = i >= kq;
    const int col = (is_v ? i - kq : i) * VEC, d = is_v ? p.dv : p.dk, head = col / d, j = col - head * d;
    T* mean = static_cast<T*>(is_v ? p.pv : p.pk) + ((cell + head) * p.pool_rows + r.row) * d + j;
    float m[VEC];
    if (fresh) {
      block_mean<T, VEC>(static_cast<const T*>(is_v ? p.v_cache : p.k_cache), bt, p.n_kv, d, head, j, block, p.pool, m, VEC);
      store_vec<T, VEC>(mean, m, VEC);
    } else {
      load_vec<T, VEC>(mean, m, VEC);
    }
    if (p.k_rows != nullptr) store_vec<T, VEC>(static_cast<T*>(is_v ? p.v_rows : p.k_rows) + (static_cast<size_t>(p.first[b]) + block) * p.n_kv * d + col, m, VEC);
  }
}

template <typename T>
static cudaError_t launch_conv_project(ConvProjectParams& p, int max_rows, cudaStream_t stream) {
  const bool wide = p.dk % 4 == 0 && p.dv % 4 == 0 && p.width % 4 == 0 && p.c_start % 4 == 0 && p.ld % 4 == 0 &&
                    p.h_hist % 4 == 0 && p.c_hist % 4 == 0 && p.state_elems % 4 == 0 && (reinterpret_cast<uintptr_t>(p.proj) & 15) == 0;
  const int vec = wide ? 4 : 2;
  const int longest = p.hl > p.cl ? p.hl : p.cl;
  // a segment is never shorter than a history, and its angles fit the table
  p.seg_len = longest - 1 > kConvSeg ? longest - 1 : kConvSeg;
  if (p.seg_len * (p.rot / 2) > kConvSeg * kMaxRot / 2) return cudaErrorInvalidValue;
  const int units = p.h_taps != nullptr ? (p.n_q + p.n_kv) * ((p.dk + vec - 1) / vec) + p.n_kv * ((p.dv + vec - 1) / vec) : 0;
  p.h_blocks = (units + kConvThreads - 1) / kConvThreads;
  const int per = kConvThreads * vec;
  const dim3 grid(p.h_blocks + (p.width + per - 1) / per, (max_rows + p.seg_len - 1) / p.seg_len, p.seqs.B);
  if (grid.y > 65535 || grid.z > 65535) return cudaErrorInvalidValue;
  return vec == 4 ? launch_pdl(conv_project_kernel<T, 4>, grid, dim3(kConvThreads), 0, stream, p)
                  : launch_pdl(conv_project_kernel<T, 2>, grid, dim3(kConvThreads), 0, stream, p);
}

}  // namespace eredu

using namespace eredu;

// Heads: h_taps [h_taps_n, n_q dk + n_kv (dk + dv)] over columns 0 ... of proj (null: none); channels: c_taps [c_taps_n, width] over
// columns from c_start (null: none). pool > 0 (decode, at most 16 rows per sequence): means of the blocks the new tokens complete.
extern "C" int eredu_conv_project(const void* proj, float* state, void* q_out, void* x_out, const float* h_taps, const float* c_taps, const float* c_bias,
                                  void* k_cache, void* v_cache, void* pk, void* pv, const float* inv_freq, const float* q_scale,
                                  const int* positions, const int* block_table, const int* page_to_slot, const int* cu_q, const long long* slots,
                                  const int* seq_lens, int ld, int state_elems, int hl, int cl, int n_q, int n_kv, int dk, int dv, int rot, int pool,
                                  int pool_rows, int h_hist, int width, int c_start, int c_hist, int batch, int q_per_seq, int max_rows,
                                  int max_pages, int fp32, cudaStream_t stream) {
  if (batch <= 0 || max_rows <= 0) return 0;
  if (rot < 0 || rot > dk || rot % 2 != 0 || rot > kMaxRot || (h_taps != nullptr && (hl < 1 || n_kv < 1 || dk < 1 || dv < 1)) || (c_taps != nullptr && cl < 1)) return -1;
  // the means are formed by the thread that appends, so a sequence's rows must be one segment; longer portions leave them to
  // eredu_pool_blocks
  const int inline_pool = cu_q == nullptr && max_rows <= kConvSeg ? pool : 0;
  if (pool > 0 && cu_q == nullptr && inline_pool == 0) return -1;
  ConvProjectParams p = {proj, state, q_out, x_out, h_taps, c_taps, c_bias, k_cache, v_cache, pk, pv, inv_freq, q_scale, positions, seq_lens,
                         {block_table, page_to_slot, cu_q, slots, batch, q_per_seq, max_pages}, ld, state_elems, hl, cl, n_q, n_kv, dk, dv, rot,
                         inline_pool, pool_rows, h_hist, width, c_start, c_hist, 0, 0};
  const cudaError_t e = fp32 ? launch_conv_project<float>(p, max_rows, stream) : launch_conv_project<__nv_bfloat16>(p, max_rows, stream);
  eredu_count_launches(1);
  return static_cast<int>(e);
}

// Means of the blocks of `pool` tokens that the new tokens of every sequence complete, into pk / pv [pages, n_kv, pool_rows, width] at the page
// of a block's last token; k_rows / v_rows (null: not wanted): all whole blocks of sequence b as dense rows from row first[b] on.
extern "C" int eredu_pool_blocks(const void* k_cache, const void* v_cache, void* pk, void* pv, void* k_rows, void* v_rows, const int* block_table,
                                 const int* seq_lens, const int* cu_q, const int* first, int batch, int max_pages, int max_blocks, int n_kv, int dk,
                                 int dv, int pool, int pool_rows, int fp32, cudaStream_t stream) {
  if (batch <= 0 || max_blocks <= 0) return 0;
  if (pool <= 0 || pool_rows < (16 + pool - 1) / pool || batch > 65535) return -1;
  const PoolParams p = {k_cache, v_cache, pk, pv, k_rows, v_rows, block_table, seq_lens, cu_q, first, max_pages, n_kv, dk, dv, pool, pool_rows};
  const dim3 grid(max_blocks, batch);
  const bool wide = dk % 8 == 0 && dv % 8 == 0;
  cudaError_t e;
  if (fp32) e = wide ? launch_pdl(pool_blocks_kernel<float, 8>, grid, dim3(128), 0, stream, p) : launch_pdl(pool_blocks_kernel<float, 1>, grid, dim3(128), 0, stream, p);
  else e = wide ? launch_pdl(pool_blocks_kernel<__nv_bfloat16, 8>, grid, dim3(128), 0, stream, p)
                : launch_pdl(pool_blocks_kernel<__nv_bfloat16, 1>, grid, dim3(128), 0, stream, p);
  eredu_count_launches(1);
  return static_cast<int>(e);
}
