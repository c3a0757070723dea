// Small steps around attention (sm_100a, bf16 or fp32):
//
//   latent_norm_cache:  RMS norms of the query latent and of the key / value latent, the latter into the paged cache, followed by a
//                       key part that is rotated by its position (neighbouring dimensions are pairs)
//   rotate_tail:        the same rotation of the last dimensions of every query head
//   gate_heads:         x <- x * sigmoid(gate), a gate per column or per group of neighbouring columns
//   talk_mix:           softmax weights mixed over heads, after the products with the values: head h of the result is
//                       sum_g talk[h, g] o[g, own key / value head of h], times sigmoid(gate)
#include "common.cuh"

namespace mfb {
namespace hmx {

__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float2 ld2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 ld2(const __nv_bfloat16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
__device__ __forceinline__ void st2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void st2(__nv_bfloat16* p, float a, float b) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b);
}
// 16-bit results take the fast exponential
template <typename T>
__device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + (sizeof(T) == 2 ? __expf(-z) : expf(-z))); }

// (u, v) turned by the angle position * freq
__device__ __forceinline__ void rotate(float& u, float& v, long long position, float freq) {
  float s, c;
  sincosf(static_cast<float>(position) * freq, &s, &c);
  const float a = u * c - v * s;
  v = v * c + u * s;
  u = a;
}

// one CTA of two warpgroups' worth of warps per token: the first half norms the query latent, the second the other one
template <typename T>
__global__ void __launch_bounds__(256)
latent_norm_cache_kernel(const T* __restrict__ proj, long long ld_proj, const T* __restrict__ q_norm, const T* __restrict__ kv_norm,
                         float eps, const int* __restrict__ slots, T* __restrict__ q, T* __restrict__ cache,
                         const float* __restrict__ freqs, const long long* __restrict__ positions, int Q, int R, int P) {
  __shared__ float red[8];
  const long long t = blockIdx.x;
  const int half = threadIdx.x >> 7, tid = threadIdx.x & 127;
  const int n = half ? R : Q;
  const T* src = proj + t * ld_proj + (half ? Q : 0);
  float ss = 0.f;
  for (int i = tid; i < n; i += 128) {
    const float v = ld(src + i);
    ss = fmaf(v, v, ss);
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  const float* r = red + half * 4;
  const float rstd = 1.f / sqrtf(((r[0] + r[1]) + (r[2] + r[3])) / n + eps);
  const int slot = slots[t];
  if (half && slot < 0) return;
  const T* w = half ? kv_norm : q_norm;
  T* dst = half ? cache + (long long)slot * (R + P) : q + t * Q;
  for (int i = tid; i < n; i += 128) st(dst + i, ld(src + i) * rstd * ld(w + i));
  if (!half) return;
  for (int i = tid; i < P / 2; i += 128) {
    float u = ld(src + R + 2 * i), v = ld(src + R + 2 * i + 1);
    rotate(u, v, positions[t], freqs[i]);
    st(dst + R + 2 * i, u);
    st(dst + R + 2 * i + 1, v);
  }
}

// a thread per pair
template <typename T>
__global__ void __launch_bounds__(256)
rotate_tail_kernel(T* __restrict__ x, const float* __restrict__ freqs, const long long* __restrict__ positions, int T_rows, int H,
                   int D, int P) {
  const int half = P / 2;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < (long long)T_rows * H * half;
       i += (long long)gridDim.x * blockDim.x) {
    const long long head = i / half;
    const int k = (int)(i % half);
    T* p = x + head * D + D - P + 2 * k;
    float u = ld(p), v = ld(p + 1);
    rotate(u, v, positions[head / H], freqs[k]);
    st(p, u);
    st(p + 1, v);
  }
}

// bf16, four pairs per thread; the heads of a token that a thread meets share its cosines
__global__ void __launch_bounds__(256)
rotate_tail_vec_kernel(__nv_bfloat16* __restrict__ x, const float* __restrict__ freqs, const long long* __restrict__ positions, int H,
                       int D, int P) {
  const long long t = blockIdx.x;
  const int per = P / 8, lanes = blockDim.x / per * per;        // threads in use: whole tails
  if ((int)threadIdx.x >= lanes) return;
  const int k = threadIdx.x % per;
  float c[4], s[4];
  const float pos = static_cast<float>(positions[t]);
#pragma unroll
  for (int i = 0; i < 4; ++i) sincosf(pos * freqs[4 * k + i], &s[i], &c[i]);
  for (int h = threadIdx.x / per; h < H; h += lanes / per) {
    uint4* p = reinterpret_cast<uint4*>(x + (t * H + h) * D + D - P + 8 * k);
    uint4 u = *p;
    __nv_bfloat162* v = reinterpret_cast<__nv_bfloat162*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 f = __bfloat1622float2(v[i]);
      v[i] = __floats2bfloat162_rn(f.x * c[i] - f.y * s[i], f.y * c[i] + f.x * s[i]);
    }
    *p = u;
  }
}

// bf16, eight columns per access, a warp per token and latent, which it keeps in registers: latents of up to 32 * 8 * kHold
constexpr int kHold = 8;
__global__ void __launch_bounds__(256)
latent_norm_cache_vec_kernel(const __nv_bfloat16* __restrict__ proj, long long ld_proj, const __nv_bfloat16* __restrict__ q_norm,
                             const __nv_bfloat16* __restrict__ kv_norm, float eps, const int* __restrict__ slots,
                             __nv_bfloat16* __restrict__ q, __nv_bfloat16* __restrict__ cache, const float* __restrict__ freqs,
                             const long long* __restrict__ positions, int T_rows, int Q, int R, int P) {
  const int unit = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (unit >= 2 * T_rows) return;
  const long long t = unit >> 1;
  const bool kv = unit & 1;
  const int n = kv ? R : Q, slot = slots[t];
  if (kv && slot < 0) return;
  const __nv_bfloat16* src = proj + t * ld_proj + (kv ? Q : 0);
  const __nv_bfloat16* w = kv ? kv_norm : q_norm;
  uint4 x[kHold];
#pragma unroll
  for (int i = 0; i < kHold; ++i) {
    const int c = (i * 32 + lane) * 8;
    x[i] = c < n ? *reinterpret_cast<const uint4*>(src + c) : make_uint4(0u, 0u, 0u, 0u);
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < kHold; ++i) {
    const __nv_bfloat162* v = reinterpret_cast<const __nv_bfloat162*>(&x[i]);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 f = __bfloat1622float2(v[e]);
      ss = fmaf(f.x, f.x, fmaf(f.y, f.y, ss));
    }
  }
  const float rstd = 1.f / sqrtf(warp_sum(ss) / n + eps);
  __nv_bfloat16* dst = kv ? cache + (long long)slot * (R + P) : q + t * Q;
  if (kv) {
    for (int i = lane; i < P / 2; i += 32) {
      float2 f = ld2(src + R + 2 * i);
      rotate(f.x, f.y, positions[t], freqs[i]);
      st2(dst + R + 2 * i, f.x, f.y);
    }
  }
#pragma unroll
  for (int i = 0; i < kHold; ++i) {
    const int c = (i * 32 + lane) * 8;
    if (c >= n) break;
    const uint4 wu = *reinterpret_cast<const uint4*>(w + c);
    const __nv_bfloat162* wv = reinterpret_cast<const __nv_bfloat162*>(&wu);
    __nv_bfloat162* v = reinterpret_cast<__nv_bfloat162*>(&x[i]);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 f = __bfloat1622float2(v[e]), g = __bfloat1622float2(wv[e]);
      v[e] = __floats2bfloat162_rn(f.x * rstd * g.x, f.y * rstd * g.y);
    }
    *reinterpret_cast<uint4*>(dst + c) = x[i];
  }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(256)
gate_heads_kernel(T* __restrict__ x, long long ld_x, const T* __restrict__ gate, long long ld_g, long long T_rows, int n, int per) {
  const int nv = n / VEC;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < T_rows * nv; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / nv;
    const int c = (int)(i % nv) * VEC;
    T* p = x + t * ld_x + c;
    const T* g = gate + t * ld_g;
    if constexpr (VEC == 2) {
      const float2 v = ld2(p);
      st2(p, v.x * sigmoid<T>(ld(g + c / per)), v.y * sigmoid<T>(ld(g + (c + 1) / per)));
    } else {
      st(p, ld(p) * sigmoid<T>(ld(g + c / per)));
    }
  }
}

// bf16, eight columns per access; PER8: the eight columns share a gate
template <bool PER8>
__global__ void __launch_bounds__(256)
gate_heads_vec_kernel(__nv_bfloat16* __restrict__ x, long long ld_x, const __nv_bfloat16* __restrict__ gate, long long ld_g, int T_rows,
                      int n, int per) {
  const int nv = n / 8;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < (long long)T_rows * nv; i += (long long)gridDim.x * blockDim.x) {
    const int t = (int)(i / nv), c = (int)(i % nv) * 8;
    uint4* p = reinterpret_cast<uint4*>(x + t * ld_x + c);
    uint4 u = *p;
    __nv_bfloat162* v = reinterpret_cast<__nv_bfloat162*>(&u);
    const __nv_bfloat16* g = gate + t * ld_g;
    float s[8];
    if constexpr (PER8) {
      s[0] = sigmoid<__nv_bfloat16>(ld(g + c / per));
#pragma unroll
      for (int k = 1; k < 8; ++k) s[k] = s[0];
    } else {
#pragma unroll
      for (int k = 0; k < 8; ++k) s[k] = sigmoid<__nv_bfloat16>(ld(g + c + k));
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const float2 f = __bfloat1622float2(v[k]);
      v[k] = __floats2bfloat162_rn(f.x * s[2 * k], f.y * s[2 * k + 1]);
    }
    *p = u;
  }
}

constexpr int kAcc = 8;

// a thread keeps up to eight result heads of one key / value head for VEC columns; the matrix lies in shared memory
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
talk_mix_kernel(const T* __restrict__ o, const float* __restrict__ talk, const T* __restrict__ gate, long long ld_g, T* __restrict__ y,
                int H, int G, int DV, int in_smem) {
  extern __shared__ float sh[];
  const long long t = blockIdx.x;
  if (in_smem) {
    for (int i = threadIdx.x; i < H * H; i += blockDim.x) sh[i] = talk[i];
    __syncthreads();
  }
  const float* tm = in_smem ? sh : talk;
  const int group = H / G, blocks = (group + kAcc - 1) / kAcc, nv = DV / VEC;
  const T* src = o + t * H * G * DV;
  for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < G * blocks * nv; i += gridDim.y * blockDim.x) {
    const int d = (i % nv) * VEC, kb = i / nv, kv = kb / blocks, h0 = kv * group + (kb % blocks) * kAcc;
    const int m = min(kAcc, kv * group + group - h0);
    float acc[kAcc][VEC];
#pragma unroll
    for (int j = 0; j < kAcc; ++j)
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[j][e] = 0.f;
    for (int g = 0; g < H; ++g) {
      float v[VEC];
      const T* p = src + ((long long)g * G + kv) * DV + d;
      if constexpr (VEC == 2) { const float2 f = ld2(p); v[0] = f.x; v[1] = f.y; }
      else v[0] = ld(p);
#pragma unroll
      for (int j = 0; j < kAcc; ++j)
        if (j < m) {
          const float w = tm[(h0 + j) * H + g];
#pragma unroll
          for (int e = 0; e < VEC; ++e) acc[j][e] = fmaf(w, v[e], acc[j][e]);
        }
    }
#pragma unroll
    for (int j = 0; j < kAcc; ++j)
      if (j < m) {
        const long long col = (long long)(h0 + j) * DV + d;
        float r[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) r[e] = gate ? acc[j][e] * sigmoid<T>(ld(gate + t * ld_g + col + e)) : acc[j][e];
        T* dst = y + t * H * DV + col;
        if constexpr (VEC == 2) st2(dst, r[0], r[1]);
        else st(dst, r[0]);
      }
  }
}

// bf16, DV a multiple of 8, up to GR heads per key / value head at a time: a thread keeps GR result heads of 8 columns. The matrix
// lies in shared memory transposed, [g][h], so that the weights of a thread's heads are one vector.
template <int GR>
__global__ void __launch_bounds__(256)
talk_mix_vec_kernel(const __nv_bfloat16* __restrict__ o, const float* __restrict__ talk, const __nv_bfloat16* __restrict__ gate,
                    long long ld_g, __nv_bfloat16* __restrict__ y, long long T, int H, int G, int DV) {
  extern __shared__ float sh[];
  const int group = H / G, blocks = (group + GR - 1) / GR, hp = G * blocks * GR;      // heads, every group padded to GR
  for (int i = threadIdx.x; i < H * hp; i += blockDim.x) {
    const int g = i / hp, p = i % hp, kv = p / (blocks * GR), r = p % (blocks * GR);
    sh[i] = r < group ? talk[(kv * group + r) * H + g] : 0.f;
  }
  __syncthreads();
  const int nv = DV / 8, per = G * blocks * nv;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < T * per; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / per;
    const int e = (int)(i % per), d = (e % nv) * 8, kb = e / nv, kv = kb / blocks;
    const __nv_bfloat16* src = o + t * H * G * DV + kv * DV + d;
    float acc[GR][8];
#pragma unroll
    for (int j = 0; j < GR; ++j)
#pragma unroll
      for (int k = 0; k < 8; ++k) acc[j][k] = 0.f;
#pragma unroll 4
    for (int g = 0; g < H; ++g) {
      const uint4 u = *reinterpret_cast<const uint4*>(src + (long long)g * G * DV);
      const __nv_bfloat162* p2 = reinterpret_cast<const __nv_bfloat162*>(&u);
      const float* w = sh + g * hp + kb * GR;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float2 f = __bfloat1622float2(p2[k]);
#pragma unroll
        for (int j = 0; j < GR; ++j) {
          acc[j][2 * k] = fmaf(w[j], f.x, acc[j][2 * k]);
          acc[j][2 * k + 1] = fmaf(w[j], f.y, acc[j][2 * k + 1]);
        }
      }
    }
#pragma unroll
    for (int j = 0; j < GR; ++j) {
      const int r = (kb % blocks) * GR + j;
      if (r < group) {
        const long long col = (long long)(kv * group + r) * DV + d;
        float v[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) v[k] = acc[j][k];
        if (gate) {
          const uint4 u = *reinterpret_cast<const uint4*>(gate + t * ld_g + col);
          const __nv_bfloat162* z = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const float2 f = __bfloat1622float2(z[k]);
            v[2 * k] *= sigmoid<__nv_bfloat16>(f.x);
            v[2 * k + 1] *= sigmoid<__nv_bfloat16>(f.y);
          }
        }
        *reinterpret_cast<uint4*>(y + t * H * DV + col) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]),
                                                                     pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
      }
    }
  }
}

bool al(const void* p, int n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; }

}  // namespace hmx
}  // namespace mfb

extern "C" {
using namespace mfb;

// proj [T, >= Q + R + P] (rows ld_proj apart): query latent | key / value latent | key part to rotate; q [T, Q]; cache rows [..,
// R + P] at slots[t] (< 0: not written); freqs [P / 2] and positions [T] (not read with P = 0). f32 = 1: all fp32, else bf16.
int mfb_latent_norm_cache(const void* proj, long long ld_proj, const void* q_norm, const void* kv_norm, float eps, const int* slots,
                          void* q, void* cache, const float* freqs, const long long* positions, int T, int Q, int R, int P, int f32,
                          cudaStream_t stream) {
  if (T <= 0) return 0;
  if (Q < 1 || R < 1 || P < 0 || P % 2 || ld_proj < Q + R + P || (P && (!freqs || !positions))) {
    mfb_host::set_error("latent_norm_cache: Q=%d R=%d P=%d", Q, R, P);
    return 1;
  }
  using bf = __nv_bfloat16;
  constexpr int most = 32 * 8 * hmx::kHold;
  if (!f32 && Q % 8 == 0 && R % 8 == 0 && P % 8 == 0 && ld_proj % 8 == 0 && Q <= most && R <= most && hmx::al(proj, 16) && hmx::al(q_norm, 16)
      && hmx::al(kv_norm, 16) && hmx::al(q, 16) && hmx::al(cache, 16)) {
    hmx::latent_norm_cache_vec_kernel<<<(int)(((long long)T * 2 + 7) / 8), 256, 0, stream>>>(
        (const bf*)proj, ld_proj, (const bf*)q_norm, (const bf*)kv_norm, eps, slots, (bf*)q, (bf*)cache, freqs,
        positions, T, Q, R, P);
    return cudaGetLastError() == cudaSuccess ? 0 : 2;
  }
  if (f32) hmx::latent_norm_cache_kernel<float><<<T, 256, 0, stream>>>((const float*)proj, ld_proj, (const float*)q_norm,
      (const float*)kv_norm, eps, slots, (float*)q, (float*)cache, freqs, positions, Q, R, P);
  else hmx::latent_norm_cache_kernel<bf><<<T, 256, 0, stream>>>((const bf*)proj, ld_proj, (const bf*)q_norm, (const bf*)kv_norm,
      eps, slots, (bf*)q, (bf*)cache, freqs, positions, Q, R, P);
  return cudaGetLastError() == cudaSuccess ? 0 : 2;
}

// x [T, H, D]: the last P dimensions of every head are rotated in place by positions[t] * freqs.
int mfb_rotate_tail(void* x, const float* freqs, const long long* positions, int T, int H, int D, int P, int f32, cudaStream_t stream) {
  if (T <= 0 || P == 0) return 0;
  if (H < 1 || P < 0 || P % 2 || P > D) { mfb_host::set_error("rotate_tail: H=%d D=%d P=%d", H, D, P); return 1; }
  if (!f32 && P % 8 == 0 && D % 8 == 0 && P <= 8 * 256 && hmx::al(x, 16)) {
    const long long want = (long long)H * (P / 8);
    const int threads = want < 256 ? (int)((want + 31) / 32 * 32) : 256;
    hmx::rotate_tail_vec_kernel<<<T, threads, 0, stream>>>((__nv_bfloat16*)x, freqs, positions, H, D, P);
    return cudaGetLastError() == cudaSuccess ? 0 : 2;
  }
  const long long want = ((long long)T * H * (P / 2) + 255) / 256;
  const int grid = (int)(want < 148 * 16 ? want : 148 * 16);
  if (f32) hmx::rotate_tail_kernel<float><<<grid, 256, 0, stream>>>((float*)x, freqs, positions, T, H, D, P);
  else hmx::rotate_tail_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>((__nv_bfloat16*)x, freqs, positions, T, H, D, P);
  return cudaGetLastError() == cudaSuccess ? 0 : 2;
}

// x [T, n] *= sigmoid(gate [T, m]) with m a divisor of n: n / m neighbouring columns share a gate.
int mfb_gate_heads(void* x, long long ld_x, const void* gate, long long ld_g, int T, int n, int m, int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (n < 1 || m < 1 || n % m) { mfb_host::set_error("gate_heads: n=%d m=%d", n, m); return 1; }
  if (!f32 && n % 8 == 0 && ld_x % 8 == 0 && hmx::al(x, 16) && (n / m == 1 || (n / m) % 8 == 0)) {
    const long long want8 = ((long long)T * (n / 8) + 255) / 256;
    const int grid8 = (int)(want8 < 148 * 16 ? want8 : 148 * 16);
    __nv_bfloat16* xp = (__nv_bfloat16*)x;
    const __nv_bfloat16* gp = (const __nv_bfloat16*)gate;
    if (n / m == 1) hmx::gate_heads_vec_kernel<false><<<grid8, 256, 0, stream>>>(xp, ld_x, gp, ld_g, T, n, 1);
    else hmx::gate_heads_vec_kernel<true><<<grid8, 256, 0, stream>>>(xp, ld_x, gp, ld_g, T, n, n / m);
    return cudaGetLastError() == cudaSuccess ? 0 : 2;
  }
  const bool vec = n % 2 == 0 && ld_x % 2 == 0 && hmx::al(x, f32 ? 8 : 4);
  const long long items = (long long)T * (vec ? n / 2 : n);
  const long long want = (items + 255) / 256;
  const int grid = (int)(want < 148 * 16 ? want : 148 * 16);
  using bf = __nv_bfloat16;
  const int per = n / m;
  if (f32) {
    if (vec) hmx::gate_heads_kernel<float, 2><<<grid, 256, 0, stream>>>((float*)x, ld_x, (const float*)gate, ld_g, T, n, per);
    else hmx::gate_heads_kernel<float, 1><<<grid, 256, 0, stream>>>((float*)x, ld_x, (const float*)gate, ld_g, T, n, per);
  } else {
    if (vec) hmx::gate_heads_kernel<bf, 2><<<grid, 256, 0, stream>>>((bf*)x, ld_x, (const bf*)gate, ld_g, T, n, per);
    else hmx::gate_heads_kernel<bf, 1><<<grid, 256, 0, stream>>>((bf*)x, ld_x, (const bf*)gate, ld_g, T, n, per);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : 2;
}

// o [T, H, G, DV], talk [H, H] fp32, gate [T, H DV] (rows ld_g apart) or null -> y [T, H DV].
int mfb_talk_mix(const void* o, const float* talk, const void* gate, long long ld_g, void* y, int T, int H, int G, int DV, int f32,
                 cudaStream_t stream) {
  if (T <= 0) return 0;
  if (G < 1 || H < 1 || H % G || DV < 1) { mfb_host::set_error("talk_mix: H=%d G=%d DV=%d", H, G, DV); return 1; }
  if (!f32 && DV % 8 == 0 && hmx::al(o, 16) && hmx::al(y, 16) && (!gate || (hmx::al(gate, 16) && ld_g % 8 == 0))) {
    const int group = H / G, gr = group <= 1 ? 1 : (group == 2 ? 2 : 4), blocks = (group + gr - 1) / gr;
    const size_t bytes = (size_t)H * G * blocks * gr * 4;
    if (bytes <= 48 * 1024) {
      const long long want = ((long long)T * G * blocks * (DV / 8) + 255) / 256;
      const int grid = (int)(want < 148 * 8 ? want : 148 * 8);
      const __nv_bfloat16 *op = (const __nv_bfloat16*)o, *gp = (const __nv_bfloat16*)gate;
      __nv_bfloat16* yp = (__nv_bfloat16*)y;
      if (gr == 1) hmx::talk_mix_vec_kernel<1><<<grid, 256, bytes, stream>>>(op, talk, gp, ld_g, yp, T, H, G, DV);
      else if (gr == 2) hmx::talk_mix_vec_kernel<2><<<grid, 256, bytes, stream>>>(op, talk, gp, ld_g, yp, T, H, G, DV);
      else hmx::talk_mix_vec_kernel<4><<<grid, 256, bytes, stream>>>(op, talk, gp, ld_g, yp, T, H, G, DV);
      return cudaGetLastError() == cudaSuccess ? 0 : 2;
    }
  }
  const bool vec = DV % 2 == 0 && hmx::al(o, f32 ? 8 : 4) && hmx::al(y, f32 ? 8 : 4);
  const int in_smem = (size_t)H * H * 4 <= 48 * 1024;
  const size_t smem = in_smem ? (size_t)H * H * 4 : 0;
  const int items = G * ((H / G + hmx::kAcc - 1) / hmx::kAcc) * (vec ? DV / 2 : DV);
  int gy = 1;
  while ((long long)T * gy < 148 * 4 && gy * 256 < items) ++gy;
  const dim3 grid(T, gy);
  using bf = __nv_bfloat16;
  if (f32) {
    if (vec) hmx::talk_mix_kernel<float, 2><<<grid, 256, smem, stream>>>((const float*)o, talk, (const float*)gate, ld_g,
        (float*)y, H, G, DV, in_smem);
    else hmx::talk_mix_kernel<float, 1><<<grid, 256, smem, stream>>>((const float*)o, talk, (const float*)gate, ld_g, (float*)y, H,
        G, DV, in_smem);
  } else {
    if (vec) hmx::talk_mix_kernel<bf, 2><<<grid, 256, smem, stream>>>((const bf*)o, talk, (const bf*)gate, ld_g, (bf*)y, H, G, DV, in_smem);
    else hmx::talk_mix_kernel<bf, 1><<<grid, 256, smem, stream>>>((const bf*)o, talk, (const bf*)gate, ld_g, (bf*)y, H, G, DV, in_smem);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : 2;
}

}  // extern "C"
