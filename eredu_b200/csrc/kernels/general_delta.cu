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
  float *red;                  // [8][4] sums of the warps: k . k, r . k, r . a u, o . o
};

__device__ __forceinline__ float delta_sum(const DeltaToken& d, int which) {
  float t = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) t += d.red[w * 4 + which];
  return t;
}
__device__ __forceinline__ void delta_part(const DeltaToken& d, int which, float v) {
  v = warp_sum_f32(v);
  if ((threadIdx.x & 31) == 0) d.red[(threadIdx.x >> 5) * 4 + which] = v;
}

// Fills `d` for row `row` of head h (256 threads). The sums r . k and r . a u, and the vectors, are there behind the next barrier.
template <typename T>
__device__ __forceinline__ void delta_token(const DeltaParams<T>& p, const DeltaToken& d, const T* row, int h) {
  const int dk = p.dk, qk = p.H * dk, vw = p.H * p.dv;
  const T* low = row + 3 * qk + 2 * vw;
  float ss = 0.f;
  for (int i = threadIdx.x; i < dk; i += 256) {
    const float k = to_f32(row[qk + h * dk + i]);
    d.k[i] = k;
    d.r[i] = to_f32(row[h * dk + i]);
    d.au[i] = sigmoid_f32(to_f32(row[2 * qk + 2 * vw + h * dk + i]) + p.rate_b[h * dk + i]);
    ss += k * k;
  }
  for (int i = threadIdx.x; i < p.rank; i += 256) d.low[i] = tanhf(to_f32(low[i]));
  delta_part(d, 0, ss);
  __syncthreads();
  const float inv = 1.f / sqrtf(delta_sum(d, 0) + kUnitEps);
  float rk = 0.f, ra = 0.f;
  for (int i = threadIdx.x; i < dk; i += 256) {
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
    const float u = d.k[i] * inv, au = d.au[i] * u;
    d.w[i] = expm1f(-p.log_decay * sigmoid_f32(z));
    d.u[i] = u;
    d.au[i] = au;
    rk = fmaf(d.r[i], d.k[i], rk);
    ra = fmaf(d.r[i], au, ra);
  }
  delta_part(d, 1, rk);
  delta_part(d, 2, ra);
  __syncthreads();
}

// Norm over the head, output gate, store. A thread brings o of column j = threadIdx.x (and 256 on) in os; ends behind a barrier.
template <typename T>
__device__ __forceinline__ void delta_store(const DeltaParams<T>& p, const DeltaToken& d, const float* os, const T* row, size_t m, int h) {
  const int qk = p.H * p.dk, vw = p.H * p.dv;
  float ss = 0.f;
  for (int j = threadIdx.x; j < p.dv; j += 256) ss += os[j] * os[j];
  delta_part(d, 3, ss);
  __syncthreads();
  const float inv = 1.f / sqrtf(delta_sum(d, 3) / static_cast<float>(p.dv) + p.eps);
  for (int j = threadIdx.x; j < p.dv; j += 256) {
    const float g = to_f32(row[2 * qk + vw + h * p.dv + j]);
    p.out[m * vw + h * p.dv + j] = from_f32<T>(os[j] * inv * p.norm_w[h * p.dv + j] * sigmoid_f32(g));
  }
}

constexpr int kStepRank = 16;        // inputs of a channel's decay a thread keeps in registers

// Decode steps and short portions, head sizes up to 128 in multiples of four: one CTA per (head, sequence), the state in registers for the
// whole portion - a thread holds NR rows of four columns. Each token takes one pass for u^T S and (r w)^T S, since
// o = (r w)^T S - (r . a u) u^T S + (r . k) v, and one for the update. TPC neighbouring threads share the decay of a key channel; what a
// token needs is on its way at once, and the weights are fetched before the dependency wait.
// DV > 0: value columns, and the rows of all threads together are the key channels; 0: any sizes.
template <typename T, int NR, int TPC, int DV>
__global__ void __launch_bounds__(256, NR <= 4 ? 4 : 2) delta_step_kernel(DeltaParams<T> p) {
  extern __shared__ float sm[];
  __shared__ float red[32];
  pdl_launch_early();
  const int dv = DV > 0 ? DV : p.dv, dk = DV > 0 ? NR * (1024 / (DV > 0 ? DV : 1)) : p.dk, h = blockIdx.x, tid = threadIdx.x;
  DeltaToken d;
  d.red = red;
  d.r = sm;
  d.k = d.r + dk;
  d.w = d.k + dk;
  d.u = d.w + dk;
  d.au = d.u + dk;
  float* part = d.au + dk;                                                 // [parts][2][dv]
  const int per_row = dv / 4, groups = 256 / per_row;
  // neighbouring row groups of a warp are summed with a shuffle where they fill it evenly
  const bool paired = per_row == 16, lone = per_row == 16 || per_row == 32;
  const int parts = paired ? 8 : groups;
  d.low = part + 2 * parts * dv;
  const int grp = tid / per_row, c = (tid % per_row) * 4;
  const bool mine = lone || grp < groups;
  const int ch = tid / TPC, sub = tid % TPC, qk = p.H * dk, vw = p.H * dv, ci = h * dk + min(ch, dk - 1);
  const bool has = ch < dk;
  // weights: nothing in the stream writes them
  const int share = (p.rank + TPC - 1) / TPC, k0 = sub * share, kn = max(0, min(share, p.rank - k0));
  const float* w2 = p.w2 + static_cast<size_t>(ci) * p.rank + k0;
  float w2r[kStepRank / TPC];
#pragma unroll
  for (int j = 0; j < kStepRank / TPC; ++j) w2r[j] = j < kn ? w2[j] : 0.f;
  const float w0 = p.w0[ci], rate_b = p.rate_b[ci], norm_w = tid < dv ? p.norm_w[h * dv + tid] : 0.f;
  // decode: nothing in front of this launch in the step writes the state or the tables, so it is fetched before the wait (an idle row fetches slot 0's)
  const bool early = p.seqs.cu_q == nullptr;
  int slot = 0;
  if (early) {
    slot = p.seqs.page_to_slot[p.seqs.block_table[static_cast<size_t>(blockIdx.y) * p.seqs.max_pages]];
    const char* base = reinterpret_cast<const char*>(p.state + (static_cast<size_t>(slot) * p.H + h) * dk * dv);
    const size_t bytes = static_cast<size_t>(dk) * dv * sizeof(float);
    for (size_t o = tid * 1024; o < bytes; o += 256 * 1024) bulk_prefetch_l2(base + o, static_cast<uint32_t>(bytes - o < 1024 ? bytes - o : 1024));
  }
  pdl_wait();
  pdl_launch_dependents();
  const RaggedSeq s = ragged_seq(p.seqs, blockIdx.y);
  if (s.rows <= 0) return;                                                 // uniform
  if (!early) slot = s.slot;
  float* st = p.state + (static_cast<size_t>(slot) * p.H + h) * dk * dv;
  float4 S[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int r = grp + i * groups;
    S[i] = mine && r < dk ? load4(st + static_cast<size_t>(r) * dv + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  for (int t = 0; t < s.rows; ++t) {
    const size_t m = static_cast<size_t>(s.row0 + t);
    const T* row = p.proj + m * p.ld;
    const T* vr = row + 2 * qk + h * dv + c;
    const float4 v = mine ? make_float4(to_f32(vr[0]), to_f32(vr[1]), to_f32(vr[2]), to_f32(vr[3])) : make_float4(0.f, 0.f, 0.f, 0.f);
    const float r0 = has ? to_f32(row[ci]) : 0.f, kv = has ? to_f32(row[qk + ci]) : 0.f;
    const float rate = has ? to_f32(row[2 * qk + 2 * vw + ci]) : 0.f, gate = tid < dv ? to_f32(row[2 * qk + vw + h * dv + tid]) : 0.f;
    for (int i = tid; i < p.rank; i += 256) d.low[i] = tanhf(to_f32(row[3 * qk + 2 * vw + i]));
    delta_part(d, 0, sub == 0 ? kv * kv : 0.f);
    __syncthreads();
    float z = 0.f;
#pragma unroll
    for (int j = 0; j < kStepRank / TPC; ++j)
      if (j < kn) z = fmaf(w2r[j], d.low[k0 + j], z);
    for (int j = kStepRank / TPC; j < kn; ++j) z = fmaf(w2[j], d.low[k0 + j], z);
#pragma unroll
    for (int o = TPC >> 1; o > 0; o >>= 1) z += __shfl_xor_sync(0xffffffffu, z, o);
    const float u0 = kv * (1.f / sqrtf(delta_sum(d, 0) + kUnitEps)), au0 = sigmoid_f32(rate + rate_b) * u0;
    if (has && sub == 0) {
      d.r[ch] = r0;
      d.k[ch] = kv;
      d.w[ch] = expm1f(-p.log_decay * sigmoid_f32(z + w0));
      d.u[ch] = u0;
      d.au[ch] = au0;
    }
    delta_part(d, 1, sub == 0 ? r0 * kv : 0.f);
    delta_part(d, 2, sub == 0 ? r0 * au0 : 0.f);
    __syncthreads();
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
      if (paired) {                                                        // every thread is here
        rec = make_float4(rec.x + __shfl_xor_sync(0xffffffffu, rec.x, 16), rec.y + __shfl_xor_sync(0xffffffffu, rec.y, 16),
                          rec.z + __shfl_xor_sync(0xffffffffu, rec.z, 16), rec.w + __shfl_xor_sync(0xffffffffu, rec.w, 16));
        o = make_float4(o.x + __shfl_xor_sync(0xffffffffu, o.x, 16), o.y + __shfl_xor_sync(0xffffffffu, o.y, 16),
                        o.z + __shfl_xor_sync(0xffffffffu, o.z, 16), o.w + __shfl_xor_sync(0xffffffffu, o.w, 16));
      }
      const int at = paired ? grp >> 1 : grp;
      if (!paired || (grp & 1) == 0) store4(part + (at * 2) * dv + c, rec);
      if (!paired || (grp & 1) == 1) store4(part + (at * 2 + 1) * dv + c, o);
    }
    __syncthreads();
    // o of the column that is this thread's
    float o = 0.f;
    if (tid < dv) {
      float rec = 0.f;
#pragma unroll 4
      for (int g = 0; g < parts; ++g) {
        rec += part[(g * 2) * dv + tid];
        o += part[(g * 2 + 1) * dv + tid];
      }
      o = fmaf(delta_sum(d, 1), to_f32(row[2 * qk + h * dv + tid]), fmaf(-delta_sum(d, 2), rec, o));
    }
    delta_part(d, 3, o * o);
    if (mine) {
      float4 rec = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
      for (int g = 0; g < parts; ++g) {
        const float4 x = load4(part + (g * 2) * dv + c);
        rec = make_float4(rec.x + x.x, rec.y + x.y, rec.z + x.z, rec.w + x.w);
      }
      const bool store = t + 1 == s.rows && s.live;
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        const int r = grp + i * groups;
        if (r >= dk) continue;
        const float w = d.w[r], au = d.au[r], k = d.k[r];
        S[i] = make_float4(S[i].x + fmaf(w, S[i].x, fmaf(-au, rec.x, k * v.x)), S[i].y + fmaf(w, S[i].y, fmaf(-au, rec.y, k * v.y)),
                           S[i].z + fmaf(w, S[i].z, fmaf(-au, rec.z, k * v.z)), S[i].w + fmaf(w, S[i].w, fmaf(-au, rec.w, k * v.w)));
        if (store) store4(st + static_cast<size_t>(r) * dv + c, S[i]);
      }
    }
    __syncthreads();
    if (tid < dv) {
      const float inv = 1.f / sqrtf(delta_sum(d, 3) / static_cast<float>(dv) + p.eps);
      p.out[m * vw + h * dv + tid] = from_f32<T>(o * inv * norm_w * sigmoid_f32(gate));
    }
  }
}

// Any head size: the state stays in memory, a thread owns columns.
template <typename T>
__global__ void __launch_bounds__(256) delta_any_kernel(DeltaParams<T> p) {
  extern __shared__ float sm[];
  __shared__ float red[32];
  pdl_launch_early();
  pdl_wait();
  pdl_launch_dependents();
  const int dk = p.dk, dv = p.dv, h = blockIdx.x;
  DeltaToken d;
  d.red = red;
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
    delta_token(p, d, row, h);
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
    delta_store(p, d, os, row, m, h);
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
#define ER_STEP(NR_, TPC_, DV_) return launch_pdl(delta_step_kernel<T, NR_, TPC_, DV_>, grid, dim3(256), smem, stream, p)
      if (p.dk == 64 && p.dv == 64) ER_STEP(4, 4, 64);
      if (p.dk == 128 && p.dv == 128) ER_STEP(16, 2, 128);
      if (rows <= 4) ER_STEP(4, 2, 0);
      if (rows <= 8) ER_STEP(8, 2, 0);
      ER_STEP(16, 2, 0);
#undef ER_STEP
    }
  }
  if (base > 48 * 1024) return cudaErrorInvalidValue;
  return launch_pdl(delta_any_kernel<T>, grid, dim3(256), base, stream, p);
}

}  // namespace eredu

using namespace eredu;

// Bytes of scratch a bf16 call over `rows` rows of `batch` sequences can use (0: the token-by-token kernel serves it).
extern "C" long long eredu_general_delta_scratch_bytes(int heads, int dk, int dv, int rank, int rows, int batch, int max_rows) {
  return delta_chunk_bytes(heads, dk, dv, rank, rows, batch, max_rows);
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
