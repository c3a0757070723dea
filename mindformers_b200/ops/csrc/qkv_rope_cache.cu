// Between the QKV projection and attention over a paged cache, in one kernel (sm_100a, bf16 or fp32): projection bias,
// per-head RMS norm of q and k (with or without a weight) and of v (without), rotary embedding of q and k, and the write of k and
// v into the paged cache.
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
  int unit_qk, unit_v;        // norms without a weight
  float amplitude, eps;
};

// values divided by their root mean square per head, a warp per head; a lane keeps its columns in registers
template <typename T>
__device__ __forceinline__ void unit_values(const Args& a, const T* row, const T* bias, long long off, T* dst) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int g = warp; g < a.G; g += kThreads / 32) {
    const T* src = row + off + (long long)g * a.DV;
    const T* b = bias ? bias + off + (long long)g * a.DV : nullptr;
    float v[2 * kMaxPairs], ss = 0.f;
#pragma unroll
    for (int k = 0; k < 2 * kMaxPairs; ++k) {
      const int d = lane + 32 * k;
      v[k] = d < a.DV ? ld(src + d) + (b ? ld(b + d) : 0.f) : 0.f;
      ss = fmaf(v[k], v[k], ss);
    }
    const float rstd = 1.f / sqrtf(warp_sum(ss) / a.DV + a.eps);
#pragma unroll
    for (int k = 0; k < 2 * kMaxPairs; ++k) {
      const int d = lane + 32 * k;
      if (d < a.DV) st(dst + (long long)g * a.DV + d, v[k] * rstd);
    }
  }
}

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
    if (nw || a.unit_qk) rstd = 1.f / sqrtf(warp_sum(ss) / D + a.eps);
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
        } else {
          x *= rstd;
          y *= rstd;
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
    if (a.unit_v) {
      unit_values(a, row, bias, off, dst);
    } else if (a.paired && n % 2 == 0) {
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

// eight neighbours (16-byte aligned)
__device__ __forceinline__ void ld8(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void ld8(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 u = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 f = __bfloat1622float2(h[i]);
    v[2 * i] = f.x; v[2 * i + 1] = f.y;
  }
}
__device__ __forceinline__ void st8(float* p, const float (&v)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void st8(__nv_bfloat16* p, const float (&v)[8]) {
  *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]),
                                            pack_bf16x2(v[6], v[7]));
}

// Head sizes 32, 64, 128 and 256 with neighbouring pairs: LPH = D / 8 lanes hold a head, eight dimensions (four pairs)
// each, so that a head is one 16-byte access per lane and a CTA works on 256 / LPH heads at a time.
template <typename T, int LPH>
__global__ void __launch_bounds__(kThreads) qkv_rope_cache_vec_kernel(const Args a) {
  extern __shared__ float sh[];
  constexpr int D = 8 * LPH, GROUPS = kThreads / LPH;
  const long long t = blockIdx.x;
  const int half = a.rot / 2;
  float* sh_cos = sh;
  float* sh_sin = sh + half;
  const int slot = a.slots[t];
  const float pos = static_cast<float>(a.positions[t]);
  const int sub = threadIdx.x / LPH, e = (threadIdx.x % LPH) * 8;
  const T* row = reinterpret_cast<const T*>(a.qkv) + t * a.ld_qkv;
  const T* bias = reinterpret_cast<const T*>(a.bias);
  // the first head of every group is on its way while the angles are evaluated
  float x[8];
  if (sub < a.H + a.G) ld8(row + (long long)sub * D + e, x);
  for (int i = threadIdx.x; i < half; i += kThreads) {
    float s, c;
    sincosf(pos * a.freqs[i], &s, &c);
    sh_cos[i] = c * a.amplitude;
    sh_sin[i] = s * a.amplitude;
  }
  __syncthreads();
  const int n_heads = a.H + a.G;
  for (int h0 = 0; h0 < n_heads; h0 += GROUPS) {
    const int h = h0 + sub;
    const bool on = h < n_heads;              // the shuffles below name every lane of the warp
    const bool is_q = h < a.H;
    float cur[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) cur[i] = on ? x[i] : 0.f;
    if (h + GROUPS < n_heads) ld8(row + (long long)(h + GROUPS) * D + e, x);
    if (on && bias) {
      float b[8];
      ld8(bias + (long long)h * D + e, b);
#pragma unroll
      for (int i = 0; i < 8; ++i) cur[i] += b[i];
    }
    const T* nw = reinterpret_cast<const T*>(is_q ? a.q_norm : a.k_norm);
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) ss = fmaf(cur[i], cur[i], ss);
#pragma unroll
    for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!on || (!is_q && slot < 0)) continue;
    if (nw || a.unit_qk) {
      const float rstd = 1.f / sqrtf(ss / D + a.eps);
      float w[8];
      if (nw) ld8(nw + e, w);
#pragma unroll
      for (int i = 0; i < 8; ++i) cur[i] = nw ? cur[i] * rstd * w[i] : cur[i] * rstd;
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int p = e / 2 + i;
      if (p < half) {
        const float c = sh_cos[p], s = sh_sin[p];
        const float u = cur[2 * i], v = cur[2 * i + 1];
        cur[2 * i] = u * c - v * s;
        cur[2 * i + 1] = v * c + u * s;
      }
    }
    T* dst = is_q ? reinterpret_cast<T*>(a.q_out) + (t * a.H + h) * D
                  : reinterpret_cast<T*>(a.key_cache) + ((long long)slot * a.G + (h - a.H)) * D;
    st8(dst + e, cur);
  }
  if (slot >= 0) {
    const int n = a.G * a.DV;
    const long long off = (long long)n_heads * D;
    T* dst = reinterpret_cast<T*>(a.value_cache) + (long long)slot * n;
    if (a.unit_v) {
      unit_values(a, row, bias, off, dst);
      return;
    }
    for (int i = threadIdx.x * 8; i < n; i += kThreads * 8) {
      float v[8];
      ld8(row + off + i, v);
      if (bias) {
        float b[8];
        ld8(bias + off + i, b);
#pragma unroll
        for (int k = 0; k < 8; ++k) v[k] += b[k];
      }
      st8(dst + i, v);
    }
  }
}

template <typename T>
bool launch_vec(const Args& a, int T_rows, size_t smem, cudaStream_t stream) {
  switch (a.D) {
    case 32: qkv_rope_cache_vec_kernel<T, 4><<<T_rows, kThreads, smem, stream>>>(a); return true;
    case 64: qkv_rope_cache_vec_kernel<T, 8><<<T_rows, kThreads, smem, stream>>>(a); return true;
    case 128: qkv_rope_cache_vec_kernel<T, 16><<<T_rows, kThreads, smem, stream>>>(a); return true;
    case 256: qkv_rope_cache_vec_kernel<T, 32><<<T_rows, kThreads, smem, stream>>>(a); return true;
    default: return false;
  }
}

bool al(const void* p, int n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; }

}  // namespace qrc
}  // namespace mfb

extern "C" {
using namespace mfb;

// f32 = 1: all typed tensors are fp32, else bf16. unit: bit 0: q and k, bit 1: v are normed without a weight (DV up to 512).
// freqs: [rot / 2] fp32; cos and sin are multiplied by `amplitude`.
int mfb_qkv_rope_cache(const void* qkv, long long ld_qkv, const void* bias, const void* q_norm, const void* k_norm, float eps,
                       const float* freqs, float amplitude, int rot, int interleaved, const long long* positions,
                       const int* slots, void* q_out, void* key_cache, void* value_cache, int T, int H, int G, int D, int DV,
                       int unit, int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H < 1 || G < 1 || D < 1 || DV < 1 || D > 64 * qrc::kMaxPairs || rot < 0 || rot > D || rot % 2 ||
      ((unit & 1) && (q_norm || k_norm)) || ((unit & 2) && DV > 64 * qrc::kMaxPairs)) {
    mfb_host::set_error("qkv_rope_cache: H=%d G=%d D=%d DV=%d rot=%d", H, G, D, DV, rot);
    return 1;
  }
  const int two = f32 ? 8 : 4;
  qrc::Args a;
  a.qkv = qkv; a.ld_qkv = ld_qkv; a.bias = bias; a.q_norm = q_norm; a.k_norm = k_norm; a.freqs = freqs;
  a.positions = positions; a.slots = slots; a.q_out = q_out; a.key_cache = key_cache; a.value_cache = value_cache;
  a.H = H; a.G = G; a.D = D; a.DV = DV; a.rot = rot; a.interleaved = interleaved; a.amplitude = amplitude; a.eps = eps;
  a.unit_qk = unit & 1; a.unit_v = (unit >> 1) & 1;
  a.paired = (D % 2 == 0 && (G * DV) % 2 == 0 && ld_qkv % 2 == 0 && qrc::al(qkv, two) && qrc::al(bias, two) &&
              qrc::al(q_out, two) && qrc::al(key_cache, two) && qrc::al(value_cache, two)) ? 1 : 0;
  const size_t smem = (size_t)rot * sizeof(float);
  const bool vec = interleaved && (G * DV) % 8 == 0 && ld_qkv % 8 == 0 && qrc::al(qkv, 16) && qrc::al(bias, 16) &&
                   qrc::al(q_norm, 16) && qrc::al(k_norm, 16) && qrc::al(q_out, 16) && qrc::al(key_cache, 16) &&
                   qrc::al(value_cache, 16);
  const bool done = vec && (f32 ? qrc::launch_vec<float>(a, T, smem, stream) : qrc::launch_vec<__nv_bfloat16>(a, T, smem, stream));
  if (done) {
    if (cudaGetLastError() != cudaSuccess) { mfb_host::set_error("qkv_rope_cache: launch failed"); return 2; }
    return 0;
  }
  if (f32) qrc::qkv_rope_cache_kernel<float><<<T, qrc::kThreads, smem, stream>>>(a);
  else qrc::qkv_rope_cache_kernel<__nv_bfloat16><<<T, qrc::kThreads, smem, stream>>>(a);
  if (cudaGetLastError() != cudaSuccess) { mfb_host::set_error("qkv_rope_cache: launch failed"); return 2; }
  return 0;
}

}  // extern "C"
