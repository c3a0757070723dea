// Attention over a paged cache for every head size, element type (bf16 or fp32) and mix of sequences (sm_100a): the path
// of 32-bit models and of head sizes that the tensor-core kernels (paged_prefill_tc.cu, paged_decode_tc.cu) do not serve.
//
// A batch is ragged: sequence b brings the rows cu_q[b] .. cu_q[b + 1] - 1, its last tokens, which are already in the
// cache; row r sits at position context_lens[b] - (cu_q[b + 1] - r). Keys are visible up to the row's own position, and
// with `chunk` > 0 only inside the row's chunk of `chunk` positions counted from 0, with `window` > 0 only the row's own and
// the `window` - 1 before it. With `all_values` a head's weights are applied to the values of every KV head. `sink` [Hq] adds
// exp(sink_h) to the softmax denominator of head h (no key, no value, not scaled). `softcap` > 0 bounds the scores: softcap *
// tanh(score / softcap).
//
// One CTA of four warps per (row, query head): a warp takes every fourth key, its lanes split the head dimension; the
// warps' online softmax states are merged through shared memory in a fixed order. All arithmetic is fp32.
#include "common.cuh"

namespace mfb {
namespace paa {

constexpr int kWarps = 4;
constexpr int kMaxPerLane = 32;         // head sizes up to 1024

__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// N: registers per lane for a head row (D, DV <= 32 N)
template <typename T, int N>
__global__ void __launch_bounds__(kWarps * 32)
paged_attention_any_kernel(const T* __restrict__ q, const T* __restrict__ key_cache, const T* __restrict__ value_cache,
                           const int* __restrict__ block_tables, const int* __restrict__ context_lens,
                           const int* __restrict__ cu_q, const float* __restrict__ sink, T* __restrict__ out, int B, int Hq,
                           int Hkv, int D, int DV, int block_size, int max_blocks, int chunk, int window, float scale, float softcap,
                           long long ld_out, float out_scale) {
  const int r = blockIdx.x, h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int b, pos;
  if (cu_q) {
    int lo = 0, hi = B - 1;                 // last sequence that starts at or before row r and is not empty there
    while (lo < hi) {
      const int mid = (lo + hi + 1) / 2;
      if (cu_q[mid] <= r) lo = mid; else hi = mid - 1;
    }
    b = lo;
    pos = context_lens[b] - (cu_q[b + 1] - r);
  } else {
    b = r;
    pos = context_lens[b] - 1;
  }
  int first = (chunk > 0 && pos >= 0) ? pos - pos % chunk : 0;
  if (window > 0 && pos - window + 1 > first) first = pos - window + 1;
  const int kvh = h / (Hq / Hkv), vheads = gridDim.z, vsel = blockIdx.z, vh = vheads > 1 ? vsel : kvh;
  const int* table = block_tables + (size_t)b * max_blocks;
  const T* qp = q + ((size_t)r * Hq + h) * D;
  float qr[N], acc[N];
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int d = lane + 32 * i;
    qr[i] = d < D ? ld(qp + d) * scale : 0.f;
    acc[i] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  for (int k = first + warp; k <= pos; k += kWarps) {
    const int blk = table[k / block_size];
    if (blk < 0) continue;                  // idle rows of a captured decode step have no blocks
    const size_t slot = (size_t)blk * block_size + k % block_size;
    const T* kp = key_cache + (slot * Hkv + kvh) * D;
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int d = lane + 32 * i;
      if (d < D) s = fmaf(qr[i], ld(kp + d), s);
    }
    s = warp_sum(s);
    if (softcap > 0.f) s = softcap * tanhf(s / softcap);
    const float m_new = fmaxf(m, s);
    const float alpha = expf(m - m_new), p = expf(s - m_new);
    l = l * alpha + p;
    m = m_new;
    const T* vp = value_cache + (slot * Hkv + vh) * DV;
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int d = lane + 32 * i;
      if (d < DV) acc[i] = fmaf(acc[i], alpha, p * ld(vp + d));
    }
  }
  __shared__ float sh_m[kWarps], sh_l[kWarps];
  __shared__ float sh_acc[kWarps][32 * N];
  if (lane == 0) { sh_m[warp] = m; sh_l[warp] = l; }
#pragma unroll
  for (int i = 0; i < N; ++i) sh_acc[warp][lane + 32 * i] = acc[i];
  __syncthreads();
  float mx = sink ? sink[h] : -INFINITY;
#pragma unroll
  for (int w = 0; w < kWarps; ++w) mx = fmaxf(mx, sh_m[w]);
  float den = sink ? expf(sink[h] - mx) : 0.f, wgt[kWarps];
#pragma unroll
  for (int w = 0; w < kWarps; ++w) {
    wgt[w] = sh_m[w] == -INFINITY ? 0.f : expf(sh_m[w] - mx);
    den += wgt[w] * sh_l[w];
  }
  const float inv = den > 0.f ? out_scale / den : 0.f;
  for (int d = threadIdx.x; d < DV; d += kWarps * 32) {
    float num = 0.f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) num += wgt[w] * sh_acc[w][d];
    st(out + r * ld_out + ((size_t)h * vheads + vsel) * DV + d, num * inv);
  }
}

template <typename T>
int launch(const void* q, const void* kc, const void* vc, const int* bt, const int* cl, const int* cu, const float* sink,
           void* out, int rows, int B, int Hq, int Hkv, int D, int DV, int bs, int mb, int chunk, int window, int all_values, float scale,
           float softcap, long long ld_out, float out_scale, cudaStream_t stream) {
  dim3 grid(rows, Hq, all_values ? Hkv : 1);
  const int n = ((D > DV ? D : DV) + 31) / 32;
#define MFB_PAA(N_)                                                                                                   \
  paged_attention_any_kernel<T, N_><<<grid, kWarps * 32, 0, stream>>>((const T*)q, (const T*)kc, (const T*)vc, bt, cl, \
                                                                      cu, sink, (T*)out, B, Hq, Hkv, D, DV, bs, mb,   \
                                                                      chunk, window, scale, softcap, ld_out, out_scale)
  if (n <= 2) MFB_PAA(2); else if (n <= 4) MFB_PAA(4); else if (n <= 8) MFB_PAA(8); 
  else if (n <= 16) MFB_PAA(16); else MFB_PAA(32);
#undef MFB_PAA
  if (cudaGetLastError() != cudaSuccess) { mfb_host::set_error("paged_attention_any: launch failed"); return 2; }
  return 0;
}

}  // namespace paa
}  // namespace mfb

extern "C" {
using namespace mfb;

// q [rows, Hq, D], caches [num_blocks, block_size, Hkv, D | DV], out [rows, Hq, DV] (rows ld_out apart): fp32 (f32 = 1) or bf16.
// cu_q [B + 1] (device) or null: one row per sequence. chunk <= 0: no chunks; window <= 0: no window; all_values: out [rows, Hq,
// Hkv, DV]; value_cache may be key_cache; sink: [Hq] fp32 or null. softcap > 0: scores become softcap * tanh(score / softcap).
// Rows of out lie ld_out elements apart; the result is multiplied by out_scale.
int mfb_paged_attention_any(const void* q, const void* key_cache, const void* value_cache, const int* block_tables,
                            const int* context_lens, const int* cu_q, const float* sink, void* out, int rows, int B, int Hq,
                            int Hkv, int D, int DV, int block_size, int max_blocks, int chunk, int window, int all_values, float scale,
                            float softcap, long long ld_out, float out_scale, int f32, cudaStream_t stream) {
  if (rows <= 0 || B <= 0) return 0;
  if (Hkv < 1 || Hq < 1 || Hq % Hkv || Hq > 65535 || Hkv > 65535 || D < 1 || DV < 1 || D > 32 * paa::kMaxPerLane ||
      DV > 32 * paa::kMaxPerLane || block_size < 1 || (!cu_q && rows != B)) {
    mfb_host::set_error("paged_attention_any: rows=%d B=%d Hq=%d Hkv=%d D=%d DV=%d block_size=%d", rows, B, Hq, Hkv, D, DV,
                        block_size);
    return 1;
  }
  return f32 ? paa::launch<float>(q, key_cache, value_cache, block_tables, context_lens, cu_q, sink, out, rows, B, Hq, Hkv, D,
                                  DV, block_size, max_blocks, chunk, window, all_values, scale, softcap, ld_out, out_scale, stream)
             : paa::launch<__nv_bfloat16>(q, key_cache, value_cache, block_tables, context_lens, cu_q, sink, out, rows, B, Hq,
                                          Hkv, D, DV, block_size, max_blocks, chunk, window, all_values, scale, softcap, ld_out,
                                          out_scale, stream);
}

}  // extern "C"
