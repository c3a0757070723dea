// Several residual streams per token (sm_100a, bf16 or fp32 activations): the step between two sub-layers in one pass.
//
//   x_t <- sum_s mix[s, t] x_s + write[t] * y          every stream from the old ones, plus the sub-layer's output y
//   u    = sum_t read[t] x_t                           the next sub-layer's input before its norm
//   h    = u / sqrt(mean(u^2) + eps) * w               RMS norm, in the activation type
//
// The streams x [T, n, W] are fp32. Before the first update they are all equal to the embedding row, which then stands in
// for them (`embedded`): nothing is materialised. The last step of a stack reads with ones and keeps no streams. A CTA
// handles one token; a thread reads its columns of every stream once, writes them once and keeps u in registers until the
// sum of squares is known: the kernel moves 2 n W fp32 values and two rows of activations per token and is bound by that.
#include "common.cuh"

namespace mfb {
namespace rstr {

struct Args {
  const void* x;            // [T, n, W] fp32, or [T, W] of type T (embedded)
  const void* y;            // [T, W] type T, or null (no update: the streams as they are)
  long long ld_y;
  const float* mix;         // [n, n] (from, to)
  const float* write;       // [n]
  const float* read;        // [n] or null (ones)
  const void* w;            // [W] type T
  float* x_out;             // [T, n, W] or null
  void* h;                  // [T, W] type T
  int W, n, embedded;
  float eps;
};

__device__ __forceinline__ void load4(const float* p, float (&v)[4]) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
__device__ __forceinline__ void load4(const __nv_bfloat16* p, float (&v)[4]) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
__device__ __forceinline__ void load4(const float* p, float (&v)[1]) { v[0] = *p; }
__device__ __forceinline__ void load4(const __nv_bfloat16* p, float (&v)[1]) { v[0] = __bfloat162float(*p); }
__device__ __forceinline__ void store4(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float (&v)[4]) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
}
__device__ __forceinline__ void store4(float* p, const float (&v)[1]) { *p = v[0]; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float (&v)[1]) { *p = __float2bfloat16_rn(v[0]); }

// N: streams held in registers (n <= N); VEC columns per access (4 or 1), K accesses per thread
template <typename T, int N, int VEC, int K>
__global__ void __launch_bounds__(512) streams_kernel(const Args a) {
  __shared__ float sm_mix[N * N], sm_write[N], sm_read[N], red[16];
  const long long t = blockIdx.x;
  const int n = a.n, W = a.W;
  for (int i = threadIdx.x; i < N * N; i += blockDim.x) {
    const int s = i / N, d = i % N;
    sm_mix[i] = (s < n && d < n && a.y) ? a.mix[s * n + d] : 0.f;
  }
  for (int i = threadIdx.x; i < N; i += blockDim.x) {
    sm_write[i] = (i < n && a.y) ? a.write[i] : 0.f;
    sm_read[i] = i < n ? (a.read ? a.read[i] : 1.f) : 0.f;
  }
  __syncthreads();
  const T* y = reinterpret_cast<const T*>(a.y) + t * a.ld_y;
  const float* x = reinterpret_cast<const float*>(a.x) + t * n * W;
  const T* e = reinterpret_cast<const T*>(a.x) + t * W;
  const int nvec = W / VEC;
  float u[K][VEC];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < K; ++k) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) u[k][i] = 0.f;
    const int c = threadIdx.x + k * blockDim.x;
    if (c < nvec) {
      const int col = c * VEC;
      float xs[N][VEC], yv[VEC];
      if (a.embedded) {
        load4(e + col, xs[0]);
#pragma unroll
        for (int s = 1; s < N; ++s)
#pragma unroll
          for (int i = 0; i < VEC; ++i) xs[s][i] = xs[0][i];
      } else {
#pragma unroll
        for (int s = 0; s < N; ++s) {
          if (s < n) load4(x + (long long)s * W + col, xs[s]);
          else {
#pragma unroll
            for (int i = 0; i < VEC; ++i) xs[s][i] = 0.f;
          }
        }
      }
      if (a.y) {
        load4(y + col, yv);
#pragma unroll
        for (int d = 0; d < N; ++d) {
          if (d < n) {
            float z[VEC];
            const float w = sm_write[d], r = sm_read[d];
#pragma unroll
            for (int i = 0; i < VEC; ++i) z[i] = w * yv[i];
#pragma unroll
            for (int s = 0; s < N; ++s) {
              const float m = sm_mix[s * N + d];
#pragma unroll
              for (int i = 0; i < VEC; ++i) z[i] = fmaf(m, xs[s][i], z[i]);
            }
#pragma unroll
            for (int i = 0; i < VEC; ++i) u[k][i] = fmaf(r, z[i], u[k][i]);
            if (a.x_out) store4(a.x_out + (t * n + d) * W + col, z);
          }
        }
      } else {
#pragma unroll
        for (int s = 0; s < N; ++s)
#pragma unroll
          for (int i = 0; i < VEC; ++i) u[k][i] = fmaf(sm_read[s], xs[s][i], u[k][i]);
      }
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss = fmaf(u[k][i], u[k][i], ss);
    }
  }
  ss = warp_sum(ss);
  const int nw = blockDim.x >> 5;
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < nw; ++i) tot += red[i];
  const float rstd = 1.f / sqrtf(tot / W + a.eps);
#pragma unroll
  for (int k = 0; k < K; ++k) {
    const int c = threadIdx.x + k * blockDim.x;
    if (c < nvec) {
      float w[VEC];
      load4(reinterpret_cast<const T*>(a.w) + c * VEC, w);
#pragma unroll
      for (int i = 0; i < VEC; ++i) w[i] = u[k][i] * rstd * w[i];
      store4(reinterpret_cast<T*>(a.h) + t * W + c * VEC, w);
    }
  }
}

template <typename T, int N>
int launch(const Args& a, int rows, bool vec, cudaStream_t stream) {
  const int nvec = vec ? a.W / 4 : a.W;
  int threads = (nvec + 31) / 32 * 32;
  if (threads > 512) threads = 512;
  // a few columns more per thread keep the CTA small, so that several tokens share an SM
  if (vec && threads == 512 && nvec <= 1024) threads = 256;
  const int k = (nvec + threads - 1) / threads;
#define MFB_RS(V_, K_) streams_kernel<T, N, V_, K_><<<rows, threads, 0, stream>>>(a)
  if constexpr (N <= 8) if (vec) {
    if (k <= 1) MFB_RS(4, 1); else if (k <= 2) MFB_RS(4, 2); else if (k <= 4) MFB_RS(4, 4);
    else if (k <= 8) MFB_RS(4, 8);
    else { mfb_host::set_error("residual_streams: width %d is above 16384", a.W); return 1; }
  }
  if (N > 8 || !vec) {
    if (k <= 4) MFB_RS(1, 4); else if (k <= 32) MFB_RS(1, 32);
    else { mfb_host::set_error("residual_streams: width %d is above 16384", a.W); return 1; }
  }
#undef MFB_RS
  if (cudaGetLastError() != cudaSuccess) { mfb_host::set_error("residual_streams: launch failed"); return 2; }
  return 0;
}

template <typename T>
int dispatch(const Args& a, int rows, bool vec, cudaStream_t stream) {
  if (a.n <= 2) return launch<T, 2>(a, rows, vec, stream);
  if (a.n <= 4) return launch<T, 4>(a, rows, vec, stream);
  if (a.n <= 8) return launch<T, 8>(a, rows, vec, stream);
  return launch<T, 16>(a, rows, false, stream);
}

bool al(const void* p, int bytes) { return (reinterpret_cast<uintptr_t>(p) & (bytes - 1)) == 0; }

}  // namespace rstr
}  // namespace mfb

extern "C" {
using namespace mfb;

// One step of n <= 16 residual streams (see the file header). x: [T, n, W] fp32, or the embedding rows [T, W] in the
// activation type (embedded); y [T, W] with row pitch ld_y, or null: no update. x_out may be x (in place) or null. f32: the
// activation type (y, w, h, embedding) is fp32, else bf16.
int mfb_residual_streams(const void* x, int embedded, const void* y, long long ld_y, const float* mix, const float* write,
                         const float* read, const void* w, float* x_out, void* h, int T, int n, int W, float eps, int f32,
                         cudaStream_t stream) {
  if (T <= 0) return 0;
  if (W <= 0 || n < 1 || n > 16 || (y && (!mix || !write))) {
    mfb_host::set_error("residual_streams: %d streams of width %d", n, W);
    return 1;
  }
  rstr::Args a{x, y, ld_y, mix, write, read, w, x_out, h, W, n, embedded, eps};
  const int act = f32 ? 16 : 8;
  const bool vec = W % 4 == 0 && (!y || ld_y % 4 == 0) && rstr::al(x, embedded ? act : 16) && rstr::al(y, act) &&
                   rstr::al(w, act) && rstr::al(x_out, 16) && rstr::al(h, act);
  return f32 ? rstr::dispatch<float>(a, T, vec, stream) : rstr::dispatch<__nv_bfloat16>(a, T, vec, stream);
}

}  // extern "C"
