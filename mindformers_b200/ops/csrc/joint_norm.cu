// Step of an fp32 residual stream whose sub-layers run side by side (sm_100a, bf16 or fp32 activations):
//
//   x' = x + y0 + y1 + base + step              (every term but x is optional)
//   h  = x' / rms(x') * w                       rms per part of the width: sqrt(mean(part^2) + eps); without w: h = x'
//   hc = h + conv(h),  conv(h)_t = sum_j k[j] h_(t - taps + 1 + j)       per channel, zeros before the sequence's start
//
// The parts of a norm do not meet, so a CTA takes one part of a run of consecutive rows and keeps the last h of every column in
// registers; it works out the taps - 1 rows in front of its first once more. x' is written to a buffer of its own, so rows that are
// read twice are the old ones. The rows in front of a portion come from `before` [slots, taps - 1, W], a portion's last ones go to
// `after`; a decode step has one row per slot and may use one buffer for both. Nothing is read for a row at position 0, so `before`
// needs no clearing. Rows of a decode step whose slot_mapping is negative leave `after` alone.
#include "common.cuh"

namespace mfb {
namespace jnt {

constexpr int kWarpsMax = 32;

struct Args {
  const float* x;            // [T, W]
  const void* y[2];          // [T, W], rows ld_y apart, or null
  long long ld_y[2];
  const float* base;         // [T, W] fp32, rows ld_b apart, or null
  long long ld_b;
  const void* step;          // [W] or null
  const void* w;             // [W] or null: no norm
  float* x_out;              // [T, W] or null
  void* h;                   // [T, W] or null
  void* hc;                  // [T, W] or null: no convolution
  const float* conv;         // [taps, W]
  const float* before;
  float* after;
  const int* cu_q;           // [B + 1] or null: row b belongs to slot b
  const int* context_lens;   // [B]
  const int* slots;          // [T]
  int T, W, B, part, taps, rows;      // columns per part, rows per CTA
  float eps;
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
  if (blockDim.x == 32) return v;
  float* r = red[turn];
  turn ^= 1;
  if ((threadIdx.x & 31) == 0) r[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) s += r[i];
  return s;
}

// VEC columns per access, K accesses per thread; TM: bound of the taps (weights are padded with zeros in front), 0: no convolution
template <typename T, int VEC, int K, int THREADS, int TM>
__global__ void __launch_bounds__(THREADS) joint_step_kernel(const Args a) {
  __shared__ float red[2][kWarpsMax];
  constexpr int kWin = TM > 1 ? TM - 1 : 1, kTaps = TM > 0 ? TM : 1;
  int turn = 0;
  const int W = a.W, nvec = a.part / VEC, c0 = blockIdx.y * a.part;
  const int r0 = blockIdx.x * a.rows, r1 = min(r0 + a.rows, a.T);
  const T* w = reinterpret_cast<const T*>(a.w);
  const T* step = reinterpret_cast<const T*>(a.step);
  int b = 0, r = r0;
  float win[kWin][K][VEC], cw[kTaps][K][VEC], wv[K][VEC], sv[K][VEC];
  const int skip = TM - a.taps;
#pragma unroll
  for (int k = 0; k < K; ++k) {
    const int c = c0 + (threadIdx.x + k * blockDim.x) * VEC;
    const bool in = threadIdx.x + k * blockDim.x < nvec;
#pragma unroll
    for (int i = 0; i < VEC; ++i) { wv[k][i] = 1.f; sv[k][i] = 0.f; }
    if (in && w) load(w + c, wv[k]);
    if (in && step) load(step + c, sv[k]);
    if constexpr (TM > 0) {
#pragma unroll
      for (int j = 0; j < TM; ++j) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) cw[j][k][i] = 0.f;
        if (in && j >= skip) load(a.conv + (long long)(j - skip) * W + c, cw[j][k]);
      }
#pragma unroll
      for (int j = 0; j < kWin; ++j)
#pragma unroll
        for (int i = 0; i < VEC; ++i) win[j][k][i] = 0.f;
    }
  }
  if constexpr (TM > 0) {
    if (a.cu_q) {
      int lo = 0, hi = a.B - 1;              // last sequence that starts at or before the first row (and is not empty there)
      while (lo < hi) {
        const int mid = (lo + hi + 1) / 2;
        if (a.cu_q[mid] <= r0) lo = mid; else hi = mid - 1;
      }
      b = lo;
      r = max(r0 - (a.taps - 1), a.cu_q[b]);
    }
  }
  const float inv_part = 1.f / a.part;
  for (; r < r1; ++r) {
    float xv[K][VEC];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < K; ++k) {
      const int c = c0 + (threadIdx.x + k * blockDim.x) * VEC;
      if (threadIdx.x + k * blockDim.x < nvec) {
        float v0[VEC], v1[VEC], v2[VEC];
        load(a.x + (long long)r * W + c, xv[k]);
        if (a.y[0]) load(reinterpret_cast<const T*>(a.y[0]) + r * a.ld_y[0] + c, v0);
        if (a.y[1]) load(reinterpret_cast<const T*>(a.y[1]) + r * a.ld_y[1] + c, v1);
        if (a.base) load(a.base + r * a.ld_b + c, v2);
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          if (a.y[0]) xv[k][i] += v0[i];
          if (a.y[1]) xv[k][i] += v1[i];
          if (a.base) xv[k][i] += v2[i];
          xv[k][i] += sv[k][i];
          ss = fmaf(xv[k][i], xv[k][i], ss);
        }
      }
    }
    const float rstd = w ? inv_sqrt(fmaf(block_sum(ss, red, turn), inv_part, a.eps)) : 1.f;
    const bool own = r >= r0;
    bool first = false, last = false, keep = false;
    if constexpr (TM > 0) {
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
    }
#pragma unroll
    for (int k = 0; k < K; ++k) {
      const int c = c0 + (threadIdx.x + k * blockDim.x) * VEC;
      if (threadIdx.x + k * blockDim.x < nvec) {
        float u[VEC];
#pragma unroll
        for (int i = 0; i < VEC; ++i) u[i] = xv[k][i] * rstd * wv[k][i];
        if (own) {
          if (a.x_out) store(a.x_out + (long long)r * W + c, xv[k]);
          if (a.h) store(reinterpret_cast<T*>(a.h) + (long long)r * W + c, u);
        }
        if constexpr (TM > 0) {
          const long long slot = (long long)b * (a.taps - 1) * W;
          if constexpr (TM > 1) {
            if (first) {
#pragma unroll
              for (int j = 0; j < TM - 1; ++j) {
                if (keep && j >= skip) load(a.before + slot + (long long)(j - skip) * W + c, win[j][k]);
                else {
#pragma unroll
                  for (int i = 0; i < VEC; ++i) win[j][k][i] = 0.f;
                }
              }
            }
          }
          if (own) {
            float o[VEC];
#pragma unroll
            for (int i = 0; i < VEC; ++i) {
              float s = cw[TM - 1][k][i] * u[i];
#pragma unroll
              for (int j = 0; j < TM - 1; ++j) s = fmaf(cw[j][k][i], win[j][k][i], s);
              o[i] = u[i] + s;
            }
            store(reinterpret_cast<T*>(a.hc) + (long long)r * W + c, o);
          }
          if constexpr (TM > 1) {
#pragma unroll
            for (int j = 0; j + 1 < TM - 1; ++j)
#pragma unroll
              for (int i = 0; i < VEC; ++i) win[j][k][i] = win[j + 1][k][i];
#pragma unroll
            for (int i = 0; i < VEC; ++i) win[TM - 2][k][i] = u[i];
            if (own && last) {
#pragma unroll
              for (int j = 0; j < TM - 1; ++j)
                if (j >= skip) store(a.after + slot + (long long)(j - skip) * W + c, win[j][k]);
            }
          }
        }
      }
    }
  }
}

bool al(const void* p, int n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; }

template <typename T, int VEC, int K, int THREADS>
void launch(const Args& a, cudaStream_t stream) {
  const int nvec = a.part / VEC, per = (nvec + K - 1) / K, threads = (per + 31) / 32 * 32;
  const dim3 grid((a.T + a.rows - 1) / a.rows, a.W / a.part);
  if (!a.hc) joint_step_kernel<T, VEC, K, THREADS, 0><<<grid, threads, 0, stream>>>(a);
  else if (a.taps <= 1) joint_step_kernel<T, VEC, K, THREADS, 1><<<grid, threads, 0, stream>>>(a);
  else if (a.taps <= 3) joint_step_kernel<T, VEC, K, THREADS, 3><<<grid, threads, 0, stream>>>(a);
  else if (a.taps <= 4) joint_step_kernel<T, VEC, K, THREADS, 4><<<grid, threads, 0, stream>>>(a);
  else joint_step_kernel<T, VEC, K, THREADS, 16><<<grid, threads, 0, stream>>>(a);
}

template <typename T, int VEC>
int pick(const Args& a, cudaStream_t stream) {
  const int nvec = a.part / VEC;
  if (nvec <= 256) launch<T, VEC, 1, 256>(a, stream);
  else if (nvec <= 1024) launch<T, VEC, 2, 512>(a, stream);
  else if (nvec <= 4096) launch<T, VEC, 4, 1024>(a, stream);
  else if (nvec <= 16384 && VEC == 1) launch<T, 1, 16, 1024>(a, stream);
  else { mfb_host::set_error("joint_step: parts of %d columns", a.part); return 1; }
  if (cudaGetLastError() != cudaSuccess) { mfb_host::set_error("joint_step: launch failed"); return 2; }
  return 0;
}

}  // namespace jnt
}  // namespace mfb

extern "C" {
using namespace mfb;

// See the head of this file. groups: parts of the norm; hc null: no convolution; up to 16 taps. x_out must not be x.
int mfb_joint_step(const float* x, const void* y0, long long ld_y0, const void* y1, long long ld_y1, const float* base,
                   long long ld_b, const void* step, const void* w, float* x_out, void* h, void* hc, const float* conv,
                   const float* before, float* after, const int* cu_q, const int* context_lens, const int* slots, int T, int W,
                   int B, int groups, int taps, float eps, int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (W < 1 || groups < 1 || W % groups || x_out == x || (hc && (!conv || taps < 1 || taps > 16 || (taps > 1 && (!before || !after)) ||
      !context_lens || !slots || B < 1 || (!cu_q && T != B)))) {
    mfb_host::set_error("joint_step: T=%d W=%d B=%d groups=%d taps=%d", T, W, B, groups, taps);
    return 1;
  }
  jnt::Args a;
  a.x = x; a.y[0] = y0; a.ld_y[0] = ld_y0; a.y[1] = y1; a.ld_y[1] = ld_y1; a.base = base; a.ld_b = ld_b; a.step = step; a.w = w;
  a.x_out = x_out; a.h = h; a.hc = hc; a.conv = conv; a.before = before; a.after = after; a.cu_q = cu_q;
  a.context_lens = context_lens; a.slots = slots;
  a.T = T; a.W = W; a.B = B; a.part = W / groups; a.taps = hc ? taps : 0; a.eps = eps;
  // rows per CTA: the rows in front of a run are worked out twice, so a few, as long as the GPU stays full
  a.rows = 1;
  if (hc && cu_q) while (a.rows < 16 && (long long)T / (a.rows * 2) * groups >= 148 * 6) a.rows *= 2;
  const int el = f32 ? 16 : 8;
  const bool vec = a.part % 4 == 0 && jnt::al(x, 16) && jnt::al(x_out, 16) && jnt::al(h, el) && jnt::al(hc, el) && jnt::al(w, el) &&
                   jnt::al(step, el) && jnt::al(conv, 16) && jnt::al(before, 16) && jnt::al(after, 16) &&
                   (!y0 || (jnt::al(y0, el) && ld_y0 % 4 == 0)) && (!y1 || (jnt::al(y1, el) && ld_y1 % 4 == 0)) &&
                   (!base || (jnt::al(base, 16) && ld_b % 4 == 0));
  using bf = __nv_bfloat16;
  if (f32) return vec ? jnt::pick<float, 4>(a, stream) : jnt::pick<float, 1>(a, stream);
  return vec ? jnt::pick<bf, 4>(a, stream) : jnt::pick<bf, 1>(a, stream);
}

}  // extern "C"
