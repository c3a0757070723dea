// Between the QKV projection and attention over a paged cache, in one kernel (sm_100a, bf16 or fp32): projection bias,
// per-head RMS norm of q and k, rotary embedding of q and k, and the write of k and v into the paged cache.
//
//   qkv [T, H * D + G * D + G * DV] (row pitch given)  ->  q_out [T, H, D]
//                                                          key_cache [slots, G, D], value_cache [slots, G, DV]
//
// One CTA per token. Angles are position * frequency in fp32, evaluated once per token and shared by all heads through
// shared memory: there is no table, hence no longest position. A warp handles a head at a time; its lanes hold the
// rotated pairs, (2i, 2i + 1) or (i, i + dims / 2), so that norm and rotation happen in registers. Rows with slot < 0
// (idle sequences of a decode batch) write no cache.
#include "common.cuh"

namespace mfb {
namespace qrc {

constexpr int kThreads = 256;
constexpr int kMaxPairs = 8;          // pairs per lane: head sizes up to 512

__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
// two neighbours (the address is a multiple of two elements)
__device__ __forceinline__ void ld2(const float* p, float& a, float& b) {
  const float2 f = *reinterpret_cast<const float2*>(p);
  a = f.x; b = f.y;
}
__device__ __forceinline__ void ld2(const __nv_bfloat16* p, float& a, float& b) {
  const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
  a = f.x; b = f.y;
}
__device__ __forceinline__ void st2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void st2(__nv_bfloat16* p, float a, float b) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b);
}

struct Args {
  const void* qkv;
  long long ld_qkv;
  const void* bias;           // [H D + G D + G DV] or null
  const void* q_norm;         // [D] or null
  const void* k_norm;         // [D] or null
  const float* freqs;         // [rot / 2]
  const long long* positions; // [T]
  const int* slots;           // [T]
  void* q_out;
  void* key_cache;
  void* value_cache;
  int H, G, D, DV, rot, interleaved, paired;   // paired: neighbours may be accessed two at a time
  float amplitude, eps;
};

template <typename T>
__global__ void __launch_bounds__(kThreads) qkv_rope_cache_kernel(const Args a) {
  extern __shared__ float sh[];                 // cos [rot / 2], sin [rot / 2]
  const long long t = blockIdx.x;
  const int half = a.rot / 2;
  float* sh_cos = sh;
  float* sh_sin = sh + half;
  const float pos = static_cast<float>(a.positions[t]);
  for (int i = threadIdx.x; i < half; i += kThreads) {
    float s, c;
    sincosf(pos * a.freqs[i], &s, &c);
    sh_cos[i] = c * a.amplitude;
    sh_sin[i] = s * a.amplitude;
  }
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int slot = a.slots[t];
  const T* row = reinterpret_cast<const T*>(a.qkv) + t * a.ld_qkv;
  const T* bias = reinterpret_cast<const T*>(a.bias);
  const int D = a.D, pairs = (D + 1) / 2;
  for (int h = warp; h < a.H + a.G; h += kThreads / 32) {
    const bool is_q = h < a.H;
    if (!is_q && slot < 0) continue;
    const T* src = row + (long long)h * D;
    const T* bsrc = bias ? bias + (long long)h * D : nullptr;
    float u[kMaxPairs], v[kMaxPairs];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < kMaxPairs; ++k) {
      u[k] = v[k] = 0.f;
      const int p = lane + 32 * k;
      if (p < pairs) {
        const int e0 = (a.interleaved || p >= half) ? 2 * p : p;
        const int e1 = (a.interleaved || p >= half) ? 2 * p + 1 : p + half;
        if (a.paired && e1 == e0 + 1) {
          ld2(src + e0, u[k], v[k]);
          if (bsrc) { float x, y; ld2(bsrc + e0, x, y); u[k] += x; v[k] += y; }
        } else {
          u[k] = ld(src + e0) + (bsrc ? ld(bsrc + e0) : 0.f);
          if (e1 < D) v[k] = ld(src + e1) + (bsrc ? ld(bsrc + e1) : 0.f);
        }
        ss = fmaf(u[k], u[k], fmaf(v[k], v[k], ss));
      }
    }
    const T* nw = reinterpret_cast<const T*>(is_q ? a.q_norm : a.k_norm);
    float rstd = 1.f;
    if (nw) rstd = 1.f / sqrtf(warp_sum(ss) / D + a.eps);
    T* dst = is_q ? reinterpret_cast<T*>(a.q_out) + (t * a.H + h) * D
                  : reinterpret_cast<T*>(a.key_cache) + ((long long)slot * a.G + (h - a.H)) * D;
#pragma unroll
    for (int k = 0; k < kMaxPairs; ++k) {
      const int p = lane + 32 * k;
      if (p < pairs) {
        const int e0 = (a.interleaved || p >= half) ? 2 * p : p;
        const int e1 = (a.interleaved || p >= half) ? 2 * p + 1 : p + half;
        float x = u[k], y = v[k];
        if (nw) {
          x = x * rstd * ld(nw + e0);
          if (e1 < D) y = y * rstd * ld(nw + e1);
        }
        if (p < half) {
          const float c = sh_cos[p], s = sh_sin[p];
          const float xr = x * c - y * s;
          y = y * c + x * s;
          x = xr;
        }
        if (a.paired && e1 == e0 + 1) {
          st2(dst + e0, x, y);
        } else {
          st(dst + e0, x);
          if (e1 < D) st(dst + e1, y);
        }
      }
    }
  }
  if (slot >= 0) {
    const int n = a.G * a.DV;
    const long long off = (long long)(a.H + a.G) * D;
    T* dst = reinterpret_cast<T*>(a.value_cache) + (long long)slot * n;
    if (a.paired && n % 2 == 0) {
      for (int i = threadIdx.x * 2; i < n; i += kThreads * 2) {
        float x, y;
        ld2(row + off + i, x, y);
        if (bias) { float bx, by; ld2(bias + off + i, bx, by); x += bx; y += by; }
        st2(dst + i, x, y);
      }
    } else {
      for (int i = threadIdx.x; i < n; i += kThreads) st(dst + i, ld(row + off + i) + (bias ? ld(bias + off + i) : 0.f));
    }
  }
}

bool al(const void* p, int n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; }

}  // namespace qrc
}  // namespace mfb

extern "C" {
using namespace mfb;

// f32 = 1: all typed tensors are fp32, else bf16. freqs: [rot / 2] fp32; cos and sin are multiplied by `amplitude`.
int mfb_qkv_rope_cache(const void* qkv, long long ld_qkv, const void* bias, const void* q_norm, const void* k_norm, float eps,
                       const float* freqs, float amplitude, int rot, int interleaved, const long long* positions,
                       const int* slots, void* q_out, void* key_cache, void* value_cache, int T, int H, int G, int D, int DV,
                       int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H < 1 || G < 1 || D < 1 || DV < 1 || D > 64 * qrc::kMaxPairs || rot < 0 || rot > D || rot % 2) {
    mfb_host::set_error("qkv_rope_cache: H=%d G=%d D=%d DV=%d rot=%d", H, G, D, DV, rot);
    return 1;
  }
  const int two = f32 ? 8 : 4;
  qrc::Args a;
  a.qkv = qkv; a.ld_qkv = ld_qkv; a.bias = bias; a.q_norm = q_norm; a.k_norm = k_norm; a.freqs = freqs;
  a.positions = positions; a.slots = slots; a.q_out = q_out; a.key_cache = key_cache; a.value_cache = value_cache;
  a.H = H; a.G = G; a.D = D; a.DV = DV; a.rot = rot; a.interleaved = interleaved; a.amplitude = amplitude; a.eps = eps;
  a.paired = (D % 2 == 0 && (G * DV) % 2 == 0 && ld_qkv % 2 == 0 && qrc::al(qkv, two) && qrc::al(bias, two) &&
              qrc::al(q_out, two) && qrc::al(key_cache, two) && qrc::al(value_cache, two)) ? 1 : 0;
  const size_t smem = (size_t)rot * sizeof(float);
  if (f32) qrc::qkv_rope_cache_kernel<float><<<T, qrc::kThreads, smem, stream>>>(a);
  else qrc::qkv_rope_cache_kernel<__nv_bfloat16><<<T, qrc::kThreads, smem, stream>>>(a);
  if (cudaGetLastError() != cudaSuccess) { mfb_host::set_error("qkv_rope_cache: launch failed"); return 2; }
  return 0;
}

}  // extern "C"
