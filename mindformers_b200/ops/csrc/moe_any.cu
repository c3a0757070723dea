// Mixture-of-experts steps for every size and for bf16 or fp32 (sm_100a), on the permutation plan of moe_ep.cu (expert
// segments padded to blocks of 128 rows):
//
//   clamped_glu:       y = g * sigmoid(alpha * g) * (u + shift) with g = min(x[:F], limit), u = clamp(x[F:], -limit, limit)
//   scatter / gather:  rows of one rank, optionally weighted; the path of 32-bit models and of widths that are not a
//                      multiple of 8
//   grouped_gemm_any:  out[rows of expert e] = a[rows of expert e] W[e] with W [E, K, N], fp32 FMA: the path of 32-bit
//                      models and of sizes that the tensor-core kernel does not take
//
// With the plan's segment fill the padding rows are skipped: a decode step touches the rows in use only.
#include "common.cuh"

namespace mfb {
namespace many {

constexpr int kBlock = 128;

__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// rows of 128-row block `blk` that are in use (0: none)
__device__ __forceinline__ int rows_in_use(int blk, const int* block_group, const int* num_blocks, const int* offsets,
                                           const int* fill) {
  if (!block_group) return kBlock;
  if (blk >= *num_blocks) return 0;
  if (!fill) return kBlock;
  const int e = block_group[blk];
  const int left = offsets[e] + fill[e] - blk * kBlock;
  return left < 0 ? 0 : (left > kBlock ? kBlock : left);
}

// 16-bit results take the fast exponential
template <typename T>
__device__ __forceinline__ float glu(float g, float u, float limit, float alpha, float shift) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  const float e = sizeof(T) == 2 ? __expf(-alpha * g) : expf(-alpha * g);
  return g / (1.f + e) * (u + shift);
}

// grid: (row block, column slice); VEC 8 (bf16, F % 8 == 0) or 1
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
clamped_glu_kernel(const T* __restrict__ x, T* __restrict__ y, int R, int F, float limit, float alpha, float shift,
                   const int* __restrict__ block_group, const int* __restrict__ num_blocks, const int* __restrict__ offsets,
                   const int* __restrict__ fill) {
  int used = rows_in_use(blockIdx.x, block_group, num_blocks, offsets, fill);
  const int r0 = blockIdx.x * kBlock;
  if (used > R - r0) used = R - r0;
  const int per = F / VEC;
  for (long long i = (long long)blockIdx.y * blockDim.x + threadIdx.x; i < (long long)used * per;
       i += (long long)gridDim.y * blockDim.x) {
    const long long r = r0 + i / per;
    const int c = (int)(i % per) * VEC;
    if constexpr (VEC == 8) {
      const uint4 a = *reinterpret_cast<const uint4*>(x + r * 2 * F + c);
      const uint4 b = *reinterpret_cast<const uint4*>(x + r * 2 * F + F + c);
      const __nv_bfloat162* ga = reinterpret_cast<const __nv_bfloat162*>(&a);
      const __nv_bfloat162* ub = reinterpret_cast<const __nv_bfloat162*>(&b);
      uint32_t o[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 g = __bfloat1622float2(ga[j]), u = __bfloat1622float2(ub[j]);
        o[j] = pack_bf16x2(glu<T>(g.x, u.x, limit, alpha, shift), glu<T>(g.y, u.y, limit, alpha, shift));
      }
      *reinterpret_cast<uint4*>(y + r * F + c) = make_uint4(o[0], o[1], o[2], o[3]);
    } else {
      st(y + r * F + c, glu<T>(ld(x + r * 2 * F + c), ld(x + r * 2 * F + F + c), limit, alpha, shift));
    }
  }
}

// copy c of token c / k goes to row write_base[expert] + rank within the expert, times weights[c] (null: 1)
template <typename T>
__global__ void __launch_bounds__(128)
scatter_kernel(const T* __restrict__ x, const long long* __restrict__ ids, const int* __restrict__ rank_in_e,
               const int* __restrict__ write_base, const float* __restrict__ weights, T* __restrict__ rows,
               int* __restrict__ dest_row, int k, int H, int E, int rows_cap) {
  const int c = blockIdx.x, e = (int)ids[c];
  const int row = e < E ? write_base[e] + rank_in_e[c] : -1;         // copies for identity experts have no row
  const bool ok = row >= 0 && row < rows_cap;
  if (threadIdx.x == 0) dest_row[c] = ok ? row : -1;
  if (!ok) return;
  const float w = weights ? weights[c] : 1.f;
  const T* src = x + (long long)(c / k) * H;
  for (int i = threadIdx.x; i < H; i += blockDim.x) st(rows + (long long)row * H + i, ld(src + i) * w);
}

template <typename T>
__global__ void __launch_bounds__(128)
gather_kernel(const T* __restrict__ rows, const int* __restrict__ dest_row, const float* __restrict__ weights,
              const long long* __restrict__ ids, const T* __restrict__ self, const T* __restrict__ extra, long long ld_extra,
              T* __restrict__ out, int k, int H, int E) {
  const long long t = blockIdx.x;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    float s = extra ? ld(extra + t * ld_extra + i) : 0.f;
    for (int j = 0; j < k; ++j) {
      const int r = dest_row[t * k + j];
      const float w = weights ? weights[t * k + j] : 1.f;
      if (r >= 0) s = fmaf(w, ld(rows + (long long)r * H + i), s);
      else if (self && ids[t * k + j] >= E) s = fmaf(w, ld(self + t * H + i), s);
    }
    st(out + t * H + i, s);
  }
}

constexpr int kTM = 64, kTN = 64, kTK = 16;

template <typename T>
__global__ void __launch_bounds__(256)
grouped_gemm_kernel(const T* __restrict__ a, const T* __restrict__ w, T* __restrict__ out, int R, int N, int K,
                    const int* __restrict__ block_group, const int* __restrict__ num_blocks, const int* __restrict__ offsets,
                    const int* __restrict__ fill) {
  const int r0 = blockIdx.y * kTM, blk = r0 / kBlock, n0 = blockIdx.x * kTN;
  const int used = rows_in_use(blk, block_group, num_blocks, offsets, fill);
  if (r0 - blk * kBlock >= used) return;
  const T* we = w + (long long)block_group[blk] * K * N;
  __shared__ float sa[kTK][kTM + 4], sw[kTK][kTN];
  const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kTK) {
    for (int i = threadIdx.x; i < kTM * kTK; i += 256) {
      const int r = i / kTK, k = i % kTK;
      sa[k][r] = (k0 + k < K && r0 + r < R) ? ld(a + (long long)(r0 + r) * K + k0 + k) : 0.f;
    }
    for (int i = threadIdx.x; i < kTK * kTN; i += 256) {
      const int k = i / kTN, c = i % kTN;
      sw[k][c] = (k0 + k < K && n0 + c < N) ? ld(we + (long long)(k0 + k) * N + n0 + c) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kTK; ++k) {
      float av[4], wv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { av[i] = sa[k][ty * 4 + i]; wv[i] = sw[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], wv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int r = r0 + ty * 4 + i, c = n0 + tx * 4 + j;
      if (r < R && c < N) st(out + (long long)r * N + c, acc[i][j]);
    }
}

bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace many
}  // namespace mfb

extern "C" {
using namespace mfb;

// x [R, 2 F] (gate | up) -> y [R, F]. block_group (with num_blocks) or null; offsets / fill or null: see rows_in_use.
int mfb_clamped_glu(const void* x, void* y, int R, int F, float limit, float alpha, float shift, const int* block_group,
                    const int* num_blocks,
                    const int* offsets, const int* fill, int f32, cudaStream_t stream) {
  if (R <= 0 || F <= 0) return 0;
  const int blocks = (R + many::kBlock - 1) / many::kBlock;
  const bool vec = !f32 && F % 8 == 0 && many::al16(x) && many::al16(y);
  long long slices = ((long long)many::kBlock * F / (vec ? 8 : 1) + 256 * 4 - 1) / (256 * 4);
  if (slices > 64) slices = 64;
  dim3 grid(blocks, (unsigned)slices);
  using bf = __nv_bfloat16;
  if (f32) many::clamped_glu_kernel<float, 1><<<grid, 256, 0, stream>>>((const float*)x, (float*)y, R, F, limit, alpha, shift,
      block_group, num_blocks, offsets, fill);
  else if (vec) many::clamped_glu_kernel<bf, 8><<<grid, 256, 0, stream>>>((const bf*)x, (bf*)y, R, F, limit, alpha, shift,
      block_group, num_blocks, offsets, fill);
  else many::clamped_glu_kernel<bf, 1><<<grid, 256, 0, stream>>>((const bf*)x, (bf*)y, R, F, limit, alpha, shift, block_group,
      num_blocks, offsets, fill);
  return cudaGetLastError() == cudaSuccess ? 0 : 2;
}

int mfb_moe_scatter_any(const void* x, const long long* ids, const int* rank_in_e, const int* write_base, const float* weights,
                        void* rows, int* dest_row, int T, int k, int H, int E, int rows_cap, int f32, cudaStream_t stream) {
  if (T <= 0 || k <= 0) return 0;
  if (f32) many::scatter_kernel<float><<<T * k, 128, 0, stream>>>((const float*)x, ids, rank_in_e, write_base, weights,
      (float*)rows, dest_row, k, H, E, rows_cap);
  else many::scatter_kernel<__nv_bfloat16><<<T * k, 128, 0, stream>>>((const __nv_bfloat16*)x, ids, rank_in_e, write_base, weights,
      (__nv_bfloat16*)rows, dest_row, k, H, E, rows_cap);
  return cudaGetLastError() == cudaSuccess ? 0 : 2;
}

// Copies with ids >= E stand for self [T, H] (null: nothing); extra [T, H] (rows ld_extra apart; null: nothing) is added.
int mfb_moe_gather_any(const void* rows, const int* dest_row, const float* weights, const long long* ids, const void* self,
                       const void* extra, long long ld_extra, void* out, int T, int k, int H, int E, int f32, cudaStream_t stream) {
  if (T <= 0) return 0;
  using bf = __nv_bfloat16;
  if (f32) many::gather_kernel<float><<<T, 128, 0, stream>>>((const float*)rows, dest_row, weights, ids, (const float*)self,
      (const float*)extra, ld_extra, (float*)out, k, H, E);
  else many::gather_kernel<bf><<<T, 128, 0, stream>>>((const bf*)rows, dest_row, weights, ids, (const bf*)self, (const bf*)extra,
      ld_extra, (bf*)out, k, H, E);
  return cudaGetLastError() == cudaSuccess ? 0 : 2;
}

// a [R, K], w [E, K, N], out [R, N], all fp32 (f32) or bf16; R a multiple of 128.
int mfb_grouped_gemm_any(const void* a, const void* w, void* out, int R, int N, int K, const int* block_group,
                         const int* num_blocks, const int* offsets, const int* fill, int f32, cudaStream_t stream) {
  if (R <= 0 || N <= 0) return 0;
  if (R % many::kBlock || R / many::kTM > 65535 || !block_group || !num_blocks) {
    mfb_host::set_error("grouped_gemm_any: R=%d N=%d K=%d", R, N, K);
    return 1;
  }
  dim3 grid((N + many::kTN - 1) / many::kTN, R / many::kTM);
  if (f32) many::grouped_gemm_kernel<float><<<grid, 256, 0, stream>>>((const float*)a, (const float*)w, (float*)out, R, N, K,
      block_group, num_blocks, offsets, fill);
  else many::grouped_gemm_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>((const __nv_bfloat16*)a, (const __nv_bfloat16*)w,
      (__nv_bfloat16*)out, R, N, K, block_group, num_blocks, offsets, fill);
  return cudaGetLastError() == cudaSuccess ? 0 : 2;
}

}  // extern "C"
