// Element-wise steps of decoders that keep a 32-bit residual stream (sm_100a), for bf16 or fp32 activations:
//
//   add_normed:  x += scale * (norm(y + bias) * w + b)      the step behind a sub-layer whose OUTPUT is normalised:
//                projection bias, layer norm or RMS norm, per-channel layer scale and residual add in one pass; writes
//                the fp32 stream and its copy in the activation type, which is the next sub-layer's input
//   norm_stream: y = norm(x) * w + b                        final norm of the fp32 stream into the activation type
//   relu2:       y = max(x, 0)^2
//   softcap:     y = cap * tanh(x / cap)                    fp32, in place
//
// One CTA per row; a thread keeps its share of the row in registers between the passes (mean, then the mean of the
// squared deviations, then the result), so every operand is read once: the kernels are bandwidth-bound.
#include "common.cuh"

namespace mfb {
namespace onorm {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

template <int VEC> __device__ __forceinline__ void load_vec(const float* p, float (&v)[VEC]) {
  if constexpr (VEC == 8) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
  } else {
    v[0] = *p;
  }
}
template <int VEC> __device__ __forceinline__ void load_vec(const __nv_bfloat16* p, float (&v)[VEC]) {
  if constexpr (VEC == 8) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 f = __bfloat1622float2(h[i]);
      v[2 * i] = f.x; v[2 * i + 1] = f.y;
    }
  } else {
    v[0] = __bfloat162float(*p);
  }
}
template <int VEC> __device__ __forceinline__ void store_vec(float* p, const float (&v)[VEC]) {
  if constexpr (VEC == 8) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
  } else {
    *p = v[0];
  }
}
template <int VEC> __device__ __forceinline__ void store_vec(__nv_bfloat16* p, const float (&v)[VEC]) {
  if constexpr (VEC == 8) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]),
                                              pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
  } else {
    *p = __float2bfloat16_rn(v[0]);
  }
}

// sum over the CTA; `red` holds one slot per warp and is free again when the call returns everywhere
__device__ __forceinline__ float cta_sum(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[warp] = v;
  __syncthreads();
  float s = 0.f;
  for (int i = 0; i < nw; ++i) s += red[i];
  return s;
}

struct Args {
  const void* y;            // [T, W] sub-layer output (add_normed), or fp32 stream (norm_stream)
  long long ld_y;
  const void* y_bias;       // [W] or null, type T
  const void* w;            // [W] type T
  const void* b;            // [W] or null, type T
  const void* scale;        // [W] or null, type T
  const void* resid;        // [T, W] fp32 (resid_f32) or type T: the stream before this step
  int resid_f32;
  float* x_out;             // [T, W] fp32 (may be resid)
  void* copy_out;           // [T, W] type T or null
  int W;
  int layer_norm;           // 1: mean is taken off; 0: RMS
  float eps;
};

// K vectors of VEC elements per thread
template <typename T, typename TY, int VEC, int K, bool ADD>
__global__ void __launch_bounds__(512) norm_kernel(const Args a) {
  __shared__ float red[16];
  const long long t = blockIdx.x;
  const int W = a.W, nvec = W / VEC;
  const TY* y = reinterpret_cast<const TY*>(a.y) + t * a.ld_y;
  float v[K][VEC];
  float r[ADD ? K : 1][VEC];
  float sum = 0.f;
#pragma unroll
  for (int k = 0; k < K; ++k) {
    const int c = threadIdx.x + k * blockDim.x;
    if (c < nvec) {
      load_vec<VEC>(y + (long long)c * VEC, v[k]);
      if constexpr (ADD) {
        if (a.resid_f32) load_vec<VEC>(reinterpret_cast<const float*>(a.resid) + t * W + c * VEC, r[k]);
        else load_vec<VEC>(reinterpret_cast<const T*>(a.resid) + t * W + c * VEC, r[k]);
      }
      if (a.y_bias) {
        float b[VEC];
        load_vec<VEC>(reinterpret_cast<const T*>(a.y_bias) + c * VEC, b);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[k][i] += b[i];
      }
#pragma unroll
      for (int i = 0; i < VEC; ++i) sum += a.layer_norm ? v[k][i] : v[k][i] * v[k][i];
    }
  }
  float mean = cta_sum(sum, red) / W, ms;
  if (a.layer_norm) {
    float dev = 0.f;
#pragma unroll
    for (int k = 0; k < K; ++k) {
      if ((int)(threadIdx.x + k * blockDim.x) < nvec) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) { const float d = v[k][i] - mean; dev = fmaf(d, d, dev); }
      }
    }
    ms = cta_sum(dev, red) / W;
  } else {
    ms = mean;
    mean = 0.f;
  }
  const float rstd = 1.f / sqrtf(ms + a.eps);
#pragma unroll
  for (int k = 0; k < K; ++k) {
    const int c = threadIdx.x + k * blockDim.x;
    if (c < nvec) {
      float w[VEC], o[VEC];
      load_vec<VEC>(reinterpret_cast<const T*>(a.w) + c * VEC, w);
#pragma unroll
      for (int i = 0; i < VEC; ++i) o[i] = (v[k][i] - mean) * rstd * w[i];
      if (a.b) {
        load_vec<VEC>(reinterpret_cast<const T*>(a.b) + c * VEC, w);
#pragma unroll
        for (int i = 0; i < VEC; ++i) o[i] += w[i];
      }
      if constexpr (ADD) {
        if (a.scale) {
          load_vec<VEC>(reinterpret_cast<const T*>(a.scale) + c * VEC, w);
#pragma unroll
          for (int i = 0; i < VEC; ++i) o[i] *= w[i];
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i) o[i] += r[k][i];
        store_vec<VEC>(a.x_out + t * W + c * VEC, o);
        if (a.copy_out) store_vec<VEC>(reinterpret_cast<T*>(a.copy_out) + t * W + c * VEC, o);
      } else {
        store_vec<VEC>(reinterpret_cast<T*>(a.copy_out) + t * W + c * VEC, o);
      }
    }
  }
}

template <typename T, typename TY, bool ADD>
int launch(const Args& a, int T_rows, bool vec, cudaStream_t stream) {
  const int nvec = vec ? a.W / 8 : a.W;
  int threads = (nvec + 31) / 32 * 32;
  if (threads > 512) threads = 512;
  if (threads < 32) threads = 32;
  const int k = (nvec + threads - 1) / threads;
#define MFB_ON(VEC_, K_) norm_kernel<T, TY, VEC_, K_, ADD><<<T_rows, threads, 0, stream>>>(a)
  if (vec) {
    if (k <= 1) MFB_ON(8, 1); else if (k <= 2) MFB_ON(8, 2); else if (k <= 4) MFB_ON(8, 4);
    else { mfb_host::set_error("output_norm: width %d is above 16384", a.W); return 1; }
  } else {
    if (k <= 2) MFB_ON(1, 2); else if (k <= 8) MFB_ON(1, 8); else if (k <= 32) MFB_ON(1, 32);
    else { mfb_host::set_error("output_norm: width %d is above 16384", a.W); return 1; }
  }
#undef MFB_ON
  if (cudaGetLastError() != cudaSuccess) { mfb_host::set_error("output_norm: launch failed"); return 2; }
  return 0;
}

bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename T>
__global__ void relu2_kernel(const T* __restrict__ x, T* __restrict__ y, long long rows, int cols, long long ldx) {
  const long long n = rows * cols;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / cols;
    const float v = fmaxf(to_f(x[r * ldx + (i - r * cols)]), 0.f);
    y[i] = from_f<T>(v * v);
  }
}
template <typename T>
__global__ void relu2_vec_kernel(const T* __restrict__ x, T* __restrict__ y, long long nvec) {
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < nvec; i += (long long)gridDim.x * blockDim.x) {
    float v[8];
    load_vec<8>(x + i * 8, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) { v[j] = fmaxf(v[j], 0.f); v[j] *= v[j]; }
    store_vec<8>(y + i * 8, v);
  }
}

__global__ void softcap_kernel(float* __restrict__ x, long long rows, int cols, long long ld, float cap) {
  const long long n = rows * cols;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / cols;
    float* p = x + r * ld + (i - r * cols);
    *p = cap * tanhf(*p / cap);
  }
}

}  // namespace onorm
}  // namespace mfb

extern "C" {
using namespace mfb;

// x_out = resid + scale * (norm(y + y_bias) * w + b); f32 = 1: T is fp32, else bf16. resid_f32: resid is the fp32 stream
// (it may be x_out), else a [T, W] tensor of type T. copy_out (type T, may be null) receives the same rows.
int mfb_add_normed(const void* y, long long ld_y, const void* y_bias, const void* w, const void* b, const void* scale,
                   const void* resid, int resid_f32, float* x_out, void* copy_out, int T, int W, int layer_norm, float eps,
                   int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (W <= 0) { mfb_host::set_error("add_normed: width %d", W); return 1; }
  onorm::Args a{y, ld_y, y_bias, w, b, scale, resid, resid_f32, x_out, copy_out, W, layer_norm, eps};
  const bool vec = W % 8 == 0 && ld_y % 8 == 0 && onorm::al16(y) && onorm::al16(y_bias) && onorm::al16(w) && onorm::al16(b) &&
                   onorm::al16(scale) && onorm::al16(resid) && onorm::al16(x_out) && onorm::al16(copy_out);
  return f32 ? onorm::launch<float, float, true>(a, T, vec, stream)
             : onorm::launch<__nv_bfloat16, __nv_bfloat16, true>(a, T, vec, stream);
}

// y = norm(x) * w + b of the fp32 stream x [T, W]; w, b and y are fp32 (f32) or bf16.
int mfb_norm_stream(const float* x, const void* w, const void* b, void* y, int T, int W, int layer_norm, float eps, int f32,
                    cudaStream_t stream) {
  if (T <= 0) return 0;
  if (W <= 0) { mfb_host::set_error("norm_stream: width %d", W); return 1; }
  onorm::Args a{x, W, nullptr, w, b, nullptr, nullptr, 1, nullptr, y, W, layer_norm, eps};
  const bool vec = W % 8 == 0 && onorm::al16(x) && onorm::al16(w) && onorm::al16(b) && onorm::al16(y);
  return f32 ? onorm::launch<float, float, false>(a, T, vec, stream)
             : onorm::launch<__nv_bfloat16, float, false>(a, T, vec, stream);
}

// y [rows, cols] (contiguous) = max(x, 0)^2 of x [rows, cols] with row pitch ldx
int mfb_relu2(const void* x, void* y, long long rows, int cols, long long ldx, int f32, cudaStream_t stream) {
  if (rows <= 0 || cols <= 0) return 0;
  const long long n = rows * cols;
  const bool vec = ldx == cols && n % 8 == 0 && onorm::al16(x) && onorm::al16(y);
  long long blocks = ((vec ? n / 8 : n) + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  if (vec) {
    if (f32) onorm::relu2_vec_kernel<float><<<(unsigned)blocks, 256, 0, stream>>>((const float*)x, (float*)y, n / 8);
    else onorm::relu2_vec_kernel<__nv_bfloat16><<<(unsigned)blocks, 256, 0, stream>>>((const __nv_bfloat16*)x, (__nv_bfloat16*)y, n / 8);
  } else {
    if (f32) onorm::relu2_kernel<float><<<(unsigned)blocks, 256, 0, stream>>>((const float*)x, (float*)y, rows, cols, ldx);
    else onorm::relu2_kernel<__nv_bfloat16><<<(unsigned)blocks, 256, 0, stream>>>((const __nv_bfloat16*)x, (__nv_bfloat16*)y, rows, cols, ldx);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : 2;
}

// x [rows, cols] fp32 with row pitch ld, in place: cap * tanh(x / cap)
int mfb_softcap(float* x, long long rows, int cols, long long ld, float cap, cudaStream_t stream) {
  if (rows <= 0 || cols <= 0) return 0;
  if (!(cap > 0.f)) { mfb_host::set_error("softcap: cap %f is not positive", cap); return 1; }
  long long blocks = (rows * cols + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  onorm::softcap_kernel<<<(unsigned)blocks, 256, 0, stream>>>(x, rows, cols, ld, cap);
  return cudaGetLastError() == cudaSuccess ? 0 : 2;
}

}  // extern "C"
