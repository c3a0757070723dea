// Steps of an fp32 residual stream with norms on both sides of every sub-layer (sm_100a, bf16 or fp32 activations):
//
//   embed:        x = scale * table[id] + (sin, cos)(position * frequency)
//   normed_step:  x' = x + y / rms(y) * (one + w_in) + step          (without y or step: without that term)
//                 u  = x' / rms(x') * (one + w_out)
//                 h  = u                                             or, shifted by a token,
//                 h  = u + (u of the sequence's token before - u) * mu
//
// rms(a) = sqrt(mean(a^2) + eps); `one` is 1 for weights stored around zero. With the shift a CTA walks over a few consecutive
// rows and works out u of the row before its first once more; x' is written to a buffer of its own, so rows that are read
// twice are the old ones. The u that precedes a portion comes from `before` [slots, W], the last one of a portion goes to
// `after` [slots, W]; a decode step has one row per slot and may use one buffer for both. A row that starts at position 0 is
// preceded by zeros, so `before` needs no clearing. Rows of a decode step whose slot_mapping is negative leave `after` alone.
#include "common.cuh"

namespace mfb {
namespace swn {

constexpr int kWarpsMax = 32;

struct Args {
  const float* x;            // [T, W]
  const void* y;             // [T, W] type T, rows ld_y apart, or null
  long long ld_y;
  const void* w_in;          // [W] or null (no y)
  const void* step;          // [W] or null
  const void* w_out;         // [W]
  float* x_out;              // [T, W] or null
  void* h;                   // [T, W]
  const void* mu;            // [W] or null: no shift
  const float* before;
  float* after;
  const int* cu_q;           // [B + 1] or null: row b belongs to slot b
  const int* context_lens;   // [B]
  const int* slots;          // [T]
  int T, W, B, rows;         // rows per CTA
  float one, eps;
};

__device__ __forceinline__ void load(const float* p, float (&v)[4]) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
__device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[4]) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
__device__ __forceinline__ void load(const float* p, float (&v)[1]) { v[0] = *p; }
__device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[1]) { v[0] = __bfloat162float(*p); }
__device__ __forceinline__ void store(float* p, const float (&v)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[4]) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
}
__device__ __forceinline__ void store(float* p, const float (&v)[1]) { *p = v[0]; }
__device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[1]) { *p = __float2bfloat16_rn(v[0]); }

// sum over the CTA; `red` is not read again before the next call's barrier because calls alternate between two buffers
__device__ __forceinline__ float block_sum(float v, float (*red)[kWarpsMax], int& turn) {
  v = warp_sum(v);
  float* r = red[turn];
  turn ^= 1;
  if ((threadIdx.x & 31) == 0) r[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) s += r[i];
  return s;
}

// VEC columns per access, K accesses per thread
template <typename T, int VEC, int K, int THREADS, bool SHIFT>
__global__ void __launch_bounds__(THREADS) normed_step_kernel(const Args a) {
  __shared__ float red[2][kWarpsMax];
  int turn = 0;
  const int W = a.W, nvec = W / VEC;
  const int r0 = blockIdx.x * a.rows, r1 = min(r0 + a.rows, a.T);
  const T* w_in = reinterpret_cast<const T*>(a.w_in);
  const T* w_out = reinterpret_cast<const T*>(a.w_out);
  const T* step = reinterpret_cast<const T*>(a.step);
  const T* mu = reinterpret_cast<const T*>(a.mu);
  int b = 0, r = r0;
  float prev[K][VEC];
  if constexpr (SHIFT) {
    if (a.cu_q) {
      int lo = 0, hi = a.B - 1;              // last sequence that starts at or before the first row (and is not empty there)
      while (lo < hi) {
        const int mid = (lo + hi + 1) / 2;
        if (a.cu_q[mid] <= r0) lo = mid; else hi = mid - 1;
      }
      b = lo;
      if (r0 > a.cu_q[b]) r = r0 - 1;        // u of the row before
    }
  }
  for (; r < r1; ++r) {
    float v[K][VEC];
    float ss = 0.f;
    if (a.y) {
      const T* y = reinterpret_cast<const T*>(a.y) + r * a.ld_y;
#pragma unroll
      for (int k = 0; k < K; ++k) {
        const int c = threadIdx.x + k * blockDim.x;
        if (c < nvec) {
          load(y + c * VEC, v[k]);
#pragma unroll
          for (int i = 0; i < VEC; ++i) ss = fmaf(v[k][i], v[k][i], ss);
        }
      }
    }
    float xv[K][VEC];
#pragma unroll
    for (int k = 0; k < K; ++k) {
      const int c = threadIdx.x + k * blockDim.x;
      if (c < nvec) load(a.x + (long long)r * W + c * VEC, xv[k]);
    }
    if (a.y) {
      const float rstd = 1.f / sqrtf(block_sum(ss, red, turn) / W + a.eps);
#pragma unroll
      for (int k = 0; k < K; ++k) {
        const int c = threadIdx.x + k * blockDim.x;
        if (c < nvec) {
          float w[VEC];
          load(w_in + c * VEC, w);
#pragma unroll
          for (int i = 0; i < VEC; ++i) xv[k][i] += v[k][i] * rstd * (a.one + w[i]);
        }
      }
    }
    ss = 0.f;
#pragma unroll
    for (int k = 0; k < K; ++k) {
      const int c = threadIdx.x + k * blockDim.x;
      if (c < nvec) {
        if (step) {
          float w[VEC];
          load(step + c * VEC, w);
#pragma unroll
          for (int i = 0; i < VEC; ++i) xv[k][i] += w[i];
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i) ss = fmaf(xv[k][i], xv[k][i], ss);
      }
    }
    const float rstd = 1.f / sqrtf(block_sum(ss, red, turn) / W + a.eps);
    bool first = false, last = false, keep = false;
    int slot = 0;
    if constexpr (SHIFT) {
      if (r >= r0) {
        if (a.cu_q) {
          while (r >= a.cu_q[b + 1]) ++b;
          first = r == a.cu_q[b];
          last = r + 1 == a.cu_q[b + 1];
          keep = a.context_lens[b] - (a.cu_q[b + 1] - r) > 0;
        } else {
          b = r;
          first = true;
          last = a.slots[r] >= 0;
          keep = a.context_lens[b] > 1;
        }
        slot = b;
      }
    }
#pragma unroll
    for (int k = 0; k < K; ++k) {
      const int c = threadIdx.x + k * blockDim.x;
      if (c < nvec) {
        float w[VEC], u[VEC];
        load(w_out + c * VEC, w);
#pragma unroll
        for (int i = 0; i < VEC; ++i) u[i] = xv[k][i] * rstd * (a.one + w[i]);
        if (!SHIFT || r >= r0) {
          if (a.x_out) store(a.x_out + (long long)r * W + c * VEC, xv[k]);
          if constexpr (SHIFT) {
            if (first) {
              if (keep) load(a.before + (long long)slot * W + c * VEC, prev[k]);
              else {
#pragma unroll
                for (int i = 0; i < VEC; ++i) prev[k][i] = 0.f;
              }
            }
            if (last) store(a.after + (long long)slot * W + c * VEC, u);
            float m[VEC], o[VEC];
            load(mu + c * VEC, m);
#pragma unroll
            for (int i = 0; i < VEC; ++i) o[i] = fmaf(prev[k][i] - u[i], m[i], u[i]);
            store(reinterpret_cast<T*>(a.h) + (long long)r * W + c * VEC, o);
          } else {
            store(reinterpret_cast<T*>(a.h) + (long long)r * W + c * VEC, u);
          }
        }
        if constexpr (SHIFT) {
#pragma unroll
          for (int i = 0; i < VEC; ++i) prev[k][i] = u[i];
        }
      }
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
embed_kernel(const long long* __restrict__ ids, const T* __restrict__ table, const long long* __restrict__ positions,
             const double* __restrict__ freqs, float* __restrict__ x, int W, long long rows, float scale) {
  const long long t = blockIdx.x;
  long long id = ids[t];
  if (id < 0 || id >= rows) id = 0;
  const double p = static_cast<double>(positions[t]);
  const T* row = table + id * W;
  for (int i = threadIdx.x; i < (W + 1) / 2; i += blockDim.x) {
    float s = 0.f, c = 0.f;
    if (freqs) {
      const double a = p * freqs[i];
      const double turns = rint(a * 0.15915494309189533577);          // whole turns
      sincosf(static_cast<float>(fma(-turns, 6.28318530717958647693, a)), &s, &c);
    }
    float v[1];
    load(row + 2 * i, v);
    x[t * W + 2 * i] = fmaf(v[0], scale, s);
    if (2 * i + 1 < W) {
      load(row + 2 * i + 1, v);
      x[t * W + 2 * i + 1] = fmaf(v[0], scale, c);
    }
  }
}

bool al(const void* p, int n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; }

template <typename T, int VEC, int K, int THREADS>
void launch(const Args& a, cudaStream_t stream) {
  const int nvec = a.W / VEC, threads = nvec < THREADS ? (nvec + 31) / 32 * 32 : THREADS;
  const int grid = (a.T + a.rows - 1) / a.rows;
  if (a.mu) normed_step_kernel<T, VEC, K, THREADS, true><<<grid, threads, 0, stream>>>(a);
  else normed_step_kernel<T, VEC, K, THREADS, false><<<grid, threads, 0, stream>>>(a);
}

template <typename T, int VEC>
int pick(const Args& a, cudaStream_t stream) {
  const int nvec = a.W / VEC;
  // with the shift a CTA's rows follow one another: more threads for fewer columns each
  if (a.mu && nvec > 256 && nvec <= 512) launch<T, VEC, 1, 512>(a, stream);
  else if (a.mu && nvec > 512 && nvec <= 1024) launch<T, VEC, 2, 512>(a, stream);
  else if (nvec <= 256) launch<T, VEC, 1, 256>(a, stream);
  else if (nvec <= 512) launch<T, VEC, 2, 256>(a, stream);
  else if (nvec <= 1024) launch<T, VEC, 4, 256>(a, stream);
  else if (nvec <= 2048) launch<T, VEC, 4, 512>(a, stream);
  else if (nvec <= 4096) launch<T, VEC, 4, 1024>(a, stream);
  else if (nvec <= 8192) launch<T, VEC, 8, 1024>(a, stream);
  else { mfb_host::set_error("normed_step: width %d", a.W); return 1; }
  if (cudaGetLastError() != cudaSuccess) { mfb_host::set_error("normed_step: launch failed"); return 2; }
  return 0;
}

}  // namespace swn
}  // namespace mfb

extern "C" {
using namespace mfb;

// ids, positions [T] int64; table [rows, W] (fp32 with f32, else bf16); freqs [ceil(W / 2)] fp64 or null; x [T, W] fp32.
int mfb_embed_stream(const long long* ids, const void* table, const long long* positions, const double* freqs, float* x, int T,
                     int W, int rows, float scale, int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (W < 1 || rows < 1) { mfb_host::set_error("embed_stream: W=%d rows=%d", W, rows); return 1; }
  if (f32) swn::embed_kernel<float><<<T, 256, 0, stream>>>(ids, (const float*)table, positions, freqs, x, W, rows, scale);
  else swn::embed_kernel<__nv_bfloat16><<<T, 256, 0, stream>>>(ids, (const __nv_bfloat16*)table, positions, freqs, x, W, rows, scale);
  return cudaGetLastError() == cudaSuccess ? 0 : 2;
}

// See the head of this file. Widths up to 8192 (32768 when rows allow 16-byte accesses). x_out must not be x.
int mfb_normed_step(const float* x, const void* y, long long ld_y, const void* w_in, const void* step, const void* w_out,
                    float* x_out, void* h, const void* mu, const float* before, float* after, const int* cu_q,
                    const int* context_lens, const int* slots, int T, int W, int B, int zero_centered, float eps, int f32,
                    cudaStream_t stream) {
  if (T <= 0) return 0;
  if (W < 1 || (y && !w_in) || (mu && (!before || !after || !context_lens || !slots || B < 1 || (!cu_q && T != B))) || x_out == x) {
    mfb_host::set_error("normed_step: T=%d W=%d B=%d", T, W, B);
    return 1;
  }
  swn::Args a;
  a.x = x; a.y = y; a.ld_y = ld_y; a.w_in = w_in; a.step = step; a.w_out = w_out; a.x_out = x_out; a.h = h; a.mu = mu;
  a.before = before; a.after = after; a.cu_q = cu_q; a.context_lens = context_lens; a.slots = slots;
  a.T = T; a.W = W; a.B = B; a.one = zero_centered ? 1.f : 0.f; a.eps = eps;
  // rows per CTA: the row before the first is worked out twice, so a few, as long as the GPU stays full
  a.rows = 1;
  if (mu && cu_q) while (a.rows < 8 && T / (a.rows * 2) >= 148 * 6) a.rows *= 2;
  const int el = f32 ? 16 : 8;
  const bool vec = W % 4 == 0 && swn::al(x, 16) && swn::al(x_out, 16) && swn::al(h, el) && swn::al(w_out, el) && swn::al(w_in, el) &&
                   swn::al(step, el) && swn::al(mu, el) && swn::al(before, 16) && swn::al(after, 16) &&
                   (!y || (swn::al(y, el) && ld_y % 4 == 0));
  using bf = __nv_bfloat16;
  if (f32) return vec ? swn::pick<float, 4>(a, stream) : swn::pick<float, 1>(a, stream);
  return vec ? swn::pick<bf, 4>(a, stream) : swn::pick<bf, 1>(a, stream);
}

}  // extern "C"
