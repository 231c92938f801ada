// Generalised delta rule: a matrix state per head that decays per key channel and forgets what it holds under the current key.
//   w = exp(-c sigmoid(W2 tanh(low) + w0)), a = sigmoid(rate + b), u = k / |k|
//   S_t = diag(w) S_{t-1} - (a u) (u^T S_{t-1}) + k v^T,  o_t = S_t^T r,  y = norm_w rms(o) sigmoid(gate)
// proj [M, 3 H dk + 2 H dv + rank] = [r | k | v | gate | rate | low]; S fp32 [slots, H, dk, dv]. Decays, rates, unit keys, scores and S
// are fp32.
#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/launch_count.h"
#include "../common/ptx.cuh"
#include "general_delta.h"

namespace eredu {

// What one token gives a head, in shared memory.
struct DeltaToken {
  float *r, *k, *w, *u, *au;   // [dk]; w: decay - 1, so that rounding factors just below one does not add up over the tokens
  float *low;                  // [rank] tanh
};

// Fills `d` for row `row` of head h; returns (r . k, r . a u). Every thread of the block takes part.
template <typename T>
__device__ __forceinline__ float2 delta_token(const DeltaParams<T>& p, const DeltaToken& d, const T* row, int h, float* red) {
  const int dk = p.dk, qk = p.H * dk, vw = p.H * p.dv, n = blockDim.x;
  const T* low = row + 3 * qk + 2 * vw;
  for (int i = threadIdx.x; i < p.rank; i += n) d.low[i] = tanhf(to_f32(low[i]));
  float ss = 0.f;
  for (int i = threadIdx.x; i < dk; i += n) {
    const float k = to_f32(row[qk + h * dk + i]);
    d.k[i] = k;
    ss += k * k;
  }
  const float inv = 1.f / sqrtf(block_sum_f32(ss, red) + kUnitEps);        // its barriers also publish low
  float rk = 0.f, ra = 0.f;
  for (int i = threadIdx.x; i < dk; i += n) {
    const int c = h * dk + i;
    const float* w2 = p.w2 + static_cast<size_t>(c) * p.rank;
    float z = p.w0[c];
    if ((p.rank & 3) == 0) {
#pragma unroll 4
      for (int j = 0; j < p.rank; j += 4) {
        const float4 w = load4(w2 + j);
        z = fmaf(w.x, d.low[j], fmaf(w.y, d.low[j + 1], fmaf(w.z, d.low[j + 2], fmaf(w.w, d.low[j + 3], z))));
      }
    } else {
      for (int j = 0; j < p.rank; ++j) z = fmaf(w2[j], d.low[j], z);
    }
    const float r = to_f32(row[c]), k = d.k[i], u = k * inv;
    const float au = sigmoid_f32(to_f32(row[2 * qk + 2 * vw + c]) + p.rate_b[c]) * u;
    d.w[i] = expm1f(-p.log_decay * sigmoid_f32(z));
    d.r[i] = r;
    d.u[i] = u;
    d.au[i] = au;
    rk = fmaf(r, k, rk);
    ra = fmaf(r, au, ra);
  }
  rk = block_sum_f32(rk, red);
  ra = block_sum_f32(ra, red);                                             // and the vectors are visible
  return make_float2(rk, ra);
}

// Norm over the head, output gate, store: os holds o of the head.
template <typename T>
__device__ __forceinline__ void delta_store(const DeltaParams<T>& p, const float* os, const T* row, size_t m, int h, float* red) {
  const int qk = p.H * p.dk, vw = p.H * p.dv;
  float ss = 0.f;
  for (int j = threadIdx.x; j < p.dv; j += blockDim.x) ss += os[j] * os[j];
  const float inv = 1.f / sqrtf(block_sum_f32(ss, red) / static_cast<float>(p.dv) + p.eps);
  for (int j = threadIdx.x; j < p.dv; j += blockDim.x) {
    const float g = to_f32(row[2 * qk + vw + h * p.dv + j]);
    p.out[m * vw + h * p.dv + j] = from_f32<T>(os[j] * inv * p.norm_w[h * p.dv + j] * sigmoid_f32(g));
  }
}

// Decode steps and short portions, head sizes up to 128 in multiples of four: one CTA per (head, sequence), the state in registers for the
// whole portion - a thread holds NR rows of four columns. Each token takes one pass for u^T S and (r w)^T S, since
// o = (r w)^T S - (r . a u) u^T S + (r . k) v, and one for the update.
template <typename T, int NR>
__global__ void __launch_bounds__(256) delta_step_kernel(DeltaParams<T> p) {
  extern __shared__ float sm[];
  __shared__ float red[8];
  pdl_launch_early();
  const int dk = p.dk, dv = p.dv, h = blockIdx.x;
  DeltaToken d;
  d.r = sm;
  d.k = d.r + dk;
  d.w = d.k + dk;
  d.u = d.w + dk;
  d.au = d.u + dk;
  float* os = d.au + dk;                                                   // [dv]
  float* part = os + dv;                                                   // [groups][2][dv]
  const int per_row = dv / 4, groups = 256 / per_row;
  d.low = part + 2 * groups * dv;
  const int grp = threadIdx.x / per_row, c = (threadIdx.x % per_row) * 4;
  const bool mine = grp < groups;
  float4 S[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
  auto load_state = [&](const float* st) {
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int r = grp + i * groups;
      if (mine && r < dk) S[i] = load4(st + static_cast<size_t>(r) * dv + c);
    }
  };
  // decode: nothing in front of this launch in the step writes the state, so it is fetched before the wait (an idle row fetches slot 0's)
  const bool early = p.seqs.cu_q == nullptr;
  if (early) {
    const int slot = p.seqs.page_to_slot[p.seqs.block_table[static_cast<size_t>(blockIdx.y) * p.seqs.max_pages]];
    const char* base = reinterpret_cast<const char*>(p.state + (static_cast<size_t>(slot) * p.H + h) * dk * dv);
    const size_t bytes = static_cast<size_t>(dk) * dv * sizeof(float);
    for (size_t o = threadIdx.x * 1024; o < bytes; o += 256 * 1024) bulk_prefetch_l2(base + o, static_cast<uint32_t>(bytes - o < 1024 ? bytes - o : 1024));
  }
  pdl_wait();
  pdl_launch_dependents();
  const RaggedSeq s = ragged_seq(p.seqs, blockIdx.y);
  if (s.rows <= 0) return;                                                 // uniform
  float* st = p.state + (static_cast<size_t>(s.slot) * p.H + h) * dk * dv;
  if (s.live) load_state(st);
  const int qk = p.H * dk;
  for (int t = 0; t < s.rows; ++t) {
    const size_t m = static_cast<size_t>(s.row0 + t);
    const T* row = p.proj + m * p.ld;
    const float2 dots = delta_token(p, d, row, h, red);
    if (mine) {
      float4 rec = make_float4(0.f, 0.f, 0.f, 0.f), o = rec;
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        const int r = grp + i * groups;
        if (r >= dk) continue;
        const float u = d.u[r], rw = fmaf(d.r[r], d.w[r], d.r[r]);
        rec = make_float4(fmaf(u, S[i].x, rec.x), fmaf(u, S[i].y, rec.y), fmaf(u, S[i].z, rec.z), fmaf(u, S[i].w, rec.w));
        o = make_float4(fmaf(rw, S[i].x, o.x), fmaf(rw, S[i].y, o.y), fmaf(rw, S[i].z, o.z), fmaf(rw, S[i].w, o.w));
      }
      store4(part + (grp * 2) * dv + c, rec);
      store4(part + (grp * 2 + 1) * dv + c, o);
    }
    __syncthreads();
    if (mine) {
      float4 rec = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int g = 0; g < groups; ++g) {
        const float4 x = load4(part + (g * 2) * dv + c);
        rec = make_float4(rec.x + x.x, rec.y + x.y, rec.z + x.z, rec.w + x.w);
      }
      const float4 v = make_float4(to_f32(row[2 * qk + h * dv + c]), to_f32(row[2 * qk + h * dv + c + 1]), to_f32(row[2 * qk + h * dv + c + 2]),
                                   to_f32(row[2 * qk + h * dv + c + 3]));
      if (grp == 0) {
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int g = 0; g < groups; ++g) {
          const float4 x = load4(part + (g * 2 + 1) * dv + c);
          o = make_float4(o.x + x.x, o.y + x.y, o.z + x.z, o.w + x.w);
        }
        store4(os + c, make_float4(fmaf(dots.x, v.x, fmaf(-dots.y, rec.x, o.x)), fmaf(dots.x, v.y, fmaf(-dots.y, rec.y, o.y)),
                                   fmaf(dots.x, v.z, fmaf(-dots.y, rec.z, o.z)), fmaf(dots.x, v.w, fmaf(-dots.y, rec.w, o.w))));
      }
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        const int r = grp + i * groups;
        if (r >= dk) continue;
        const float w = d.w[r], au = d.au[r], k = d.k[r];
        S[i] = make_float4(S[i].x + fmaf(w, S[i].x, fmaf(-au, rec.x, k * v.x)), S[i].y + fmaf(w, S[i].y, fmaf(-au, rec.y, k * v.y)),
                           S[i].z + fmaf(w, S[i].z, fmaf(-au, rec.z, k * v.z)), S[i].w + fmaf(w, S[i].w, fmaf(-au, rec.w, k * v.w)));
      }
    }
    __syncthreads();
    delta_store(p, os, row, m, h, red);
    __syncthreads();
  }
  if (s.live && mine)
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int r = grp + i * groups;
      if (r < dk) store4(st + static_cast<size_t>(r) * dv + c, S[i]);
    }
}

// Any head size: the state stays in memory, a thread owns columns.
template <typename T>
__global__ void __launch_bounds__(256) delta_any_kernel(DeltaParams<T> p) {
  extern __shared__ float sm[];
  __shared__ float red[8];
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int dk = p.dk, dv = p.dv, h = blockIdx.x;
  DeltaToken d;
  d.r = sm;
  d.k = d.r + dk;
  d.w = d.k + dk;
  d.u = d.w + dk;
  d.au = d.u + dk;
  float* os = d.au + dk;
  d.low = os + dv;
  const RaggedSeq s = ragged_seq(p.seqs, blockIdx.y);
  if (s.rows <= 0) return;                                                 // uniform
  float* st = p.state + (static_cast<size_t>(s.slot) * p.H + h) * dk * dv;
  const int qk = p.H * dk;
  for (int t = 0; t < s.rows; ++t) {
    const size_t m = static_cast<size_t>(s.row0 + t);
    const T* row = p.proj + m * p.ld;
    delta_token(p, d, row, h, red);
    for (int j = threadIdx.x; j < dv; j += 256) {
      const float v = to_f32(row[2 * qk + h * dv + j]);
      float rec = 0.f, o = 0.f;
      if (s.live)
        for (int i = 0; i < dk; ++i) rec = fmaf(d.u[i], st[static_cast<size_t>(i) * dv + j], rec);
      for (int i = 0; i < dk; ++i) {
        float* cell = st + static_cast<size_t>(i) * dv + j;
        const float old = s.live ? *cell : 0.f;
        const float x = old + fmaf(d.w[i], old, fmaf(-d.au[i], rec, d.k[i] * v));
        if (s.live) *cell = x;
        o = fmaf(d.r[i], x, o);
      }
      os[j] = o;
    }
    __syncthreads();
    delta_store(p, os, row, m, h, red);
    __syncthreads();
  }
}

template <typename T>
static cudaError_t launch_delta_step(const DeltaParams<T>& p, cudaStream_t stream) {
  const dim3 grid(p.H, p.seqs.B);
  if (grid.y > 65535) return cudaErrorInvalidValue;
  const size_t base = (static_cast<size_t>(5) * p.dk + p.dv + p.rank) * sizeof(float);
  if (p.dv % 4 == 0 && p.dv <= 128 && p.dk <= 128 && p.dk % 4 == 0) {
    const int groups = 256 / (p.dv / 4), rows = (p.dk + groups - 1) / groups;
    const size_t smem = base + static_cast<size_t>(2) * groups * p.dv * sizeof(float);
    if (smem <= 48 * 1024) {
      if (rows <= 4) return launch_pdl(delta_step_kernel<T, 4>, grid, dim3(256), smem, stream, p);
      if (rows <= 8) return launch_pdl(delta_step_kernel<T, 8>, grid, dim3(256), smem, stream, p);
      return launch_pdl(delta_step_kernel<T, 16>, grid, dim3(256), smem, stream, p);
    }
  }
  if (base > 48 * 1024) return cudaErrorInvalidValue;
  return launch_pdl(delta_any_kernel<T>, grid, dim3(256), base, stream, p);
}

}  // namespace eredu

using namespace eredu;

// Bytes of scratch a bf16 call over `rows` rows of `batch` sequences can use (0: the token-by-token kernel serves it).
extern "C" long long eredu_general_delta_scratch_bytes(int heads, int dk, int dv, int rows, int batch, int max_rows) {
  return delta_chunk_bytes(heads, dk, dv, rows, batch, max_rows);
}

// scratch: [eredu_general_delta_scratch_bytes(...)] of a bf16 call whose rows are whole 16-byte pieces, or null (token by token).
extern "C" int eredu_general_delta(const void* proj, const float* w2, const float* w0, const float* rate_b, const float* norm_w, float* state, void* out,
                                   void* scratch, const int* block_table, const int* page_to_slot, const int* cu_q, const long long* slots,
                                   int heads, int dk, int dv, int rank, int ld, int batch, int q_per_seq, int max_rows, int max_pages,
                                   int fp32, float log_decay, float eps, cudaStream_t stream) {
  if (batch <= 0 || max_rows <= 0) return 0;
  if (heads <= 0 || dk <= 0 || dv <= 0 || rank <= 0 || log_decay <= 0.f) return -1;
  const RaggedBatch r = {block_table, page_to_slot, cu_q, slots, batch, q_per_seq, max_pages};
  cudaError_t e;
  if (fp32) {
    const DeltaParams<float> p = {static_cast<const float*>(proj), w2, w0, rate_b, norm_w, state, static_cast<float*>(out), heads, dk, dv, rank, ld,
                                  log_decay, eps, r};
    e = launch_delta_step(p, stream);
  } else {
    const DeltaParams<__nv_bfloat16> p = {static_cast<const __nv_bfloat16*>(proj), w2, w0, rate_b, norm_w, state, static_cast<__nv_bfloat16*>(out),
                                          heads, dk, dv, rank, ld, log_decay, eps, r};
    e = scratch != nullptr && delta_chunk_supported(p) ? launch_delta_chunks(p, max_rows, scratch, stream) : launch_delta_step(p, stream);
  }
  eredu_count_launches(1);
  return static_cast<int>(e);
}
