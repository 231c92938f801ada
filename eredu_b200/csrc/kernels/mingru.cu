// minGRU recurrence: gates that read only the current token, a linear recurrence per channel, an output gate.
//   z = sigmoid(proj_z), c = u + 1/2 (u >= 0) or sigmoid(u) (u < 0), S <- (1 - z) S + z c, y = S silu(g)
// proj [M, 3 width] = [z | u | g]; S fp32 [slots, width]. All gate arithmetic and S are fp32.
//
// Because a step is affine in S, a segment of tokens is one affine map: a tile of 128 tokens is cut into segments that are
// composed in parallel (a thread holds one channel of one segment in registers), the maps are chained through shared
// memory, and every segment is then replayed from its entering state. Long portions do their tiles in parallel: one launch
// writes the map of every tile, a second one chains the maps in front of its tile and replays it.
#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/launch_count.h"
#include "../common/ptx.cuh"
#include "../common/ragged.cuh"

namespace eredu {

template <typename T>
struct MinGruParams {
  const T* proj;
  float* state;
  T* out;
  int width, ld;
  RaggedBatch seqs;
  float2* maps;   // [tiles][width] (a, b) of S -> a S + b; entry 0 of a sequence is its state when the call began
};

template <typename T>
__device__ __forceinline__ float sigmoid_of(float x) {
  return sizeof(T) == 4 ? sigmoid_f32(x) : sigmoid_fast(x);
}
// a step of the recurrence as S -> a S + b
template <typename T>
__device__ __forceinline__ void mingru_step(float z_in, float u, float& a, float& b) {
  const float z = sigmoid_of<T>(z_in);
  a = 1.f - z;
  b = z * (u >= 0.f ? u + 0.5f : sigmoid_of<T>(u));
}

// Decode steps and short portions: one thread per channel, token after token.
template <typename T>
__global__ void __launch_bounds__(128) mingru_step_kernel(MinGruParams<T> p) {
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const RaggedSeq s = ragged_seq(p.seqs, blockIdx.y);
  const int c = blockIdx.x * 128 + threadIdx.x;
  if (c >= p.width || s.rows <= 0) return;
  float* st = p.state + static_cast<size_t>(s.slot) * p.width + c;
  float S = s.live ? *st : 0.f;
  for (int t = 0; t < s.rows; ++t) {
    const T* r = p.proj + static_cast<size_t>(s.row0 + t) * p.ld + c;
    float a, b;
    mingru_step<T>(to_f32(r[0]), to_f32(r[p.width]), a, b);
    S = a * S + b;
    p.out[static_cast<size_t>(s.row0 + t) * p.width + c] = from_f32<T>(S * to_f32(r[2 * p.width]) * sigmoid_of<T>(to_f32(r[2 * p.width])));
  }
  if (s.live) *st = S;
}

constexpr int kSegs = 16;   // segments a tile is cut into
constexpr int kSegLen = 8;  // tokens of a segment
constexpr int kTileTokens = kSegs * kSegLen;

template <typename T>
__global__ void __launch_bounds__(32 * kSegs) mingru_scan_kernel(MinGruParams<T> p) {
  __shared__ float sa[kSegs][32], sb[kSegs][32], carry[32];
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const RaggedSeq s = ragged_seq(p.seqs, blockIdx.y);
  if (s.rows <= 0) return;  // uniform
  const int lane = threadIdx.x & 31, seg = threadIdx.x >> 5;
  const int c = blockIdx.x * 32 + lane;
  const bool in = c < p.width;
  float* st = p.state + static_cast<size_t>(s.slot) * p.width + (in ? c : 0);
  if (seg == 0) carry[lane] = in && s.live ? *st : 0.f;
  T zr[kSegLen], ur[kSegLen], gr[kSegLen];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < kSegLen; ++i) {
      const int t = t0 + seg * kSegLen + i;
      if (in && t < s.rows) {
        const T* r = p.proj + static_cast<size_t>(s.row0 + t) * p.ld + c;
        zr[i] = r[0];
        ur[i] = r[p.width];
        gr[i] = r[2 * p.width];
      } else {
        zr[i] = ur[i] = gr[i] = from_f32<T>(0.f);
      }
    }
  };
  fetch(0);
  for (int t0 = 0; t0 < s.rows; t0 += kTileTokens) {
    float a[kSegLen], b[kSegLen], g[kSegLen];
    float A = 1.f, B = 0.f;
#pragma unroll
    for (int i = 0; i < kSegLen; ++i) {
      if (t0 + seg * kSegLen + i < s.rows) mingru_step<T>(to_f32(zr[i]), to_f32(ur[i]), a[i], b[i]);
      else a[i] = 1.f, b[i] = 0.f;  // behind the portion: the state stays
      g[i] = to_f32(gr[i]) * sigmoid_of<T>(to_f32(gr[i]));
      A *= a[i];
      B = a[i] * B + b[i];
    }
    if (t0 + kTileTokens < s.rows) fetch(t0 + kTileTokens);  // in flight while the segments are chained
    sa[seg][lane] = A;
    sb[seg][lane] = B;
    __syncthreads();
    float S = carry[lane];
    for (int j = 0; j < seg; ++j) S = sa[j][lane] * S + sb[j][lane];
    __syncthreads();  // every thread has read the carry and the maps of this tile
#pragma unroll
    for (int i = 0; i < kSegLen; ++i) {
      const int t = t0 + seg * kSegLen + i;
      S = a[i] * S + b[i];
      if (in && t < s.rows) p.out[static_cast<size_t>(s.row0 + t) * p.width + c] = from_f32<T>(S * g[i]);
    }
    if (seg == kSegs - 1) carry[lane] = S;
  }
  __syncthreads();
  if (seg == 0 && in && s.live) *st = carry[lane];
}

__device__ __forceinline__ int tile_id(const RaggedSeq& s, int b, int tile) { return s.row0 / kTileTokens + 2 * b + tile; }

// Long portions, first launch: the map of every tile but the last.
template <typename T>
__global__ void __launch_bounds__(32 * kSegs) mingru_maps_kernel(MinGruParams<T> p) {
  __shared__ float sa[kSegs][32], sb[kSegs][32];
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.z, tile = blockIdx.y;
  const RaggedSeq s = ragged_seq(p.seqs, b);
  if (s.rows <= 0 || tile * kTileTokens >= s.rows) return;  // uniform
  const int lane = threadIdx.x & 31, seg = threadIdx.x >> 5;
  const int c = blockIdx.x * 32 + lane;
  const bool in = c < p.width;
  if (tile == 0 && seg == 0 && in)
    p.maps[static_cast<size_t>(tile_id(s, b, 0)) * p.width + c] =
        make_float2(0.f, s.live ? p.state[static_cast<size_t>(s.slot) * p.width + c] : 0.f);
  if ((tile + 1) * kTileTokens >= s.rows) return;            // nothing comes after the last tile
  float A = 1.f, B = 0.f;
  if (in) {
    const T* r = p.proj + static_cast<size_t>(s.row0 + tile * kTileTokens + seg * kSegLen) * p.ld + c;
    T zr[kSegLen], ur[kSegLen];
#pragma unroll
    for (int i = 0; i < kSegLen; ++i) {
      zr[i] = r[static_cast<size_t>(i) * p.ld];
      ur[i] = r[static_cast<size_t>(i) * p.ld + p.width];
    }
#pragma unroll
    for (int i = 0; i < kSegLen; ++i) {
      float a, bb;
      mingru_step<T>(to_f32(zr[i]), to_f32(ur[i]), a, bb);
      A *= a;
      B = a * B + bb;
    }
  }
  sa[seg][lane] = A;
  sb[seg][lane] = B;
  __syncthreads();
  if (seg == 0 && in) {
    for (int j = 1; j < kSegs; ++j) {
      B = sa[j][lane] * B + sb[j][lane];
      A *= sa[j][lane];
    }
    p.maps[static_cast<size_t>(tile_id(s, b, tile + 1)) * p.width + c] = make_float2(A, B);
  }
}

// Second launch: the entering state of the tile from the maps in front of it, then the tile itself.
template <typename T>
__global__ void __launch_bounds__(32 * kSegs) mingru_tiles_kernel(MinGruParams<T> p) {
  __shared__ float sa[kSegs][32], sb[kSegs][32], ea[kSegs][32], eb[kSegs][32];
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.z, tile = blockIdx.y;
  const RaggedSeq s = ragged_seq(p.seqs, b);
  if (s.rows <= 0 || tile * kTileTokens >= s.rows) return;  // uniform
  const int lane = threadIdx.x & 31, seg = threadIdx.x >> 5;
  const int c = blockIdx.x * 32 + lane;
  const bool in = c < p.width;
  const int t0 = tile * kTileTokens + seg * kSegLen;
  T zr[kSegLen], ur[kSegLen], gr[kSegLen];
#pragma unroll
  for (int i = 0; i < kSegLen; ++i) {
    zr[i] = ur[i] = gr[i] = from_f32<T>(0.f);
    if (in && t0 + i < s.rows) {
      const T* r = p.proj + static_cast<size_t>(s.row0 + t0 + i) * p.ld + c;
      zr[i] = r[0];
      ur[i] = r[p.width];
      gr[i] = r[2 * p.width];
    }
  }
  // maps 0 .. tile, a contiguous share per segment
  const int share = (tile + kSegs) / kSegs;
  float A = 1.f, B = 0.f;
  if (in) {
    const float2* m = p.maps + static_cast<size_t>(tile_id(s, b, 0)) * p.width + c;
#pragma unroll 4
    for (int j = seg * share; j < min((seg + 1) * share, tile + 1); ++j) {
      const float2 x = m[static_cast<size_t>(j) * p.width];
      A *= x.x;
      B = x.x * B + x.y;
    }
  }
  ea[seg][lane] = A;
  eb[seg][lane] = B;
  float a[kSegLen], bb[kSegLen];
  A = 1.f;
  B = 0.f;
#pragma unroll
  for (int i = 0; i < kSegLen; ++i) {
    if (t0 + i < s.rows) mingru_step<T>(to_f32(zr[i]), to_f32(ur[i]), a[i], bb[i]);
    else a[i] = 1.f, bb[i] = 0.f;
    A *= a[i];
    B = a[i] * B + bb[i];
  }
  sa[seg][lane] = A;
  sb[seg][lane] = B;
  __syncthreads();
  float S = 0.f;
#pragma unroll
  for (int j = 0; j < kSegs; ++j) S = ea[j][lane] * S + eb[j][lane];   // entry 0 forgets what was before it
  for (int j = 0; j < seg; ++j) S = sa[j][lane] * S + sb[j][lane];
#pragma unroll
  for (int i = 0; i < kSegLen; ++i) {
    S = a[i] * S + bb[i];
    if (in && t0 + i < s.rows) {
      const float g = to_f32(gr[i]);
      p.out[static_cast<size_t>(s.row0 + t0 + i) * p.width + c] = from_f32<T>(S * (g * sigmoid_of<T>(g)));
    }
  }
  if (seg == kSegs - 1 && in && s.live && (tile + 1) * kTileTokens >= s.rows) p.state[static_cast<size_t>(s.slot) * p.width + c] = S;
}

// Portions up to here take the single launch that walks its tiles.
constexpr int kWalkTokens = 2 * kTileTokens;
static long long mingru_tile_count(int rows, int batch) { return (rows + kTileTokens - 1) / kTileTokens + 2LL * batch; }

template <typename T>
static cudaError_t launch_mingru(const MinGruParams<T>& p, int max_rows, cudaStream_t stream) {
  if (max_rows <= 8) return launch_pdl(mingru_step_kernel<T>, dim3((p.width + 127) / 128, p.seqs.B), dim3(128), 0, stream, p);
  if (max_rows > kWalkTokens && p.maps != nullptr) {
    const dim3 grid((p.width + 31) / 32, (max_rows + kTileTokens - 1) / kTileTokens, p.seqs.B);
    if (grid.y > 65535) return cudaErrorInvalidValue;
    const cudaError_t e = launch_pdl(mingru_maps_kernel<T>, grid, dim3(32 * kSegs), 0, stream, p);
    if (e != cudaSuccess) return e;
    eredu_count_launches(1);
    return launch_pdl(mingru_tiles_kernel<T>, grid, dim3(32 * kSegs), 0, stream, p);
  }
  return launch_pdl(mingru_scan_kernel<T>, dim3((p.width + 31) / 32, p.seqs.B), dim3(32 * kSegs), 0, stream, p);
}

}  // namespace eredu

using namespace eredu;

// fp32 elements of scratch a call over `rows` rows of `batch` sequences can use (0: none).
extern "C" long long eredu_mingru_scratch_elems(int width, int rows, int batch, int max_rows) {
  return max_rows > kWalkTokens ? mingru_tile_count(rows, batch) * width * 2 : 0;
}

// scratch: fp32 [eredu_mingru_scratch_elems(...)] or null.
extern "C" int eredu_mingru_scan(const void* proj, float* state, void* out, float* scratch, const int* block_table, const int* page_to_slot,
                                 const int* cu_q, const long long* slots, int width, int ld, int batch, int q_per_seq, int max_rows,
                                 int max_pages, int fp32, cudaStream_t stream) {
  if (batch <= 0 || width <= 0 || max_rows <= 0) return 0;
  const RaggedBatch r = {block_table, page_to_slot, cu_q, slots, batch, q_per_seq, max_pages};
  cudaError_t e;
  if (fp32) {
    MinGruParams<float> p = {static_cast<const float*>(proj), state, static_cast<float*>(out), width, ld, r, reinterpret_cast<float2*>(scratch)};
    e = launch_mingru(p, max_rows, stream);
  } else {
    MinGruParams<__nv_bfloat16> p = {static_cast<const __nv_bfloat16*>(proj), state, static_cast<__nv_bfloat16*>(out), width, ld, r, reinterpret_cast<float2*>(scratch)};
    e = launch_mingru(p, max_rows, stream);
  }
  eredu_count_launches(1);
  return static_cast<int>(e);
}
