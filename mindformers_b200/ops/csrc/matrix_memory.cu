// Matrix memory with exponential gating (the mLSTM recurrence) over ragged batches (sm_100a, bf16 or fp32 activations).
//
// Per head, with q, k of size D, v of size DV and log gates i = cap tanh((x_i + b_i) / cap), f = log_sigmoid(cap tanh((x_f +
// b_f) / cap)):
//   m' = max(f + m, i);  S' = e^(f + m - m') S + e^(i - m') k v^T;  n' = e^(f + m - m') n + e^(i - m') k
//   o  = S'^T q / (max(|n' . q|, e^(-m')) + 1e-6)        with q scaled by D^(-1/2)
// and the result is o / rms(o) * norm * sigmoid(gate), rms over a head's DV columns. A row of the projection holds
// q | k | v | gate | x_i | x_f. S [slots, H, D, DV], n [slots, H, D], m [slots, H] are fp32; row b of a batch uses slot b. A
// sequence that starts at position 0 reads none of them, so a slot changes hands without being cleared.
//
//   scan_kernel:   portions, token by token on the FMA pipes; a CTA holds 32 columns of one head's S in registers
//   finish_kernel: norm, gate and the new n and m of the scan (which other CTAs of it read until then)
//   decode_kernel: one row per slot, all in one pass; rows of idle slots (slot_mapping < 0) become zeros
#include "common.cuh"

namespace mfb {
namespace mmem {

__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

__device__ __forceinline__ float input_gate(float x, float cap) { return cap * tanhf(x / cap); }
__device__ __forceinline__ float forget_gate(float x, float cap) {
  const float z = cap * tanhf(x / cap);
  return fminf(z, 0.f) - log1pf(expf(-fabsf(z)));
}

struct Args {
  const void* proj;          // [T, >= 2 H (D + DV) + 2 H]
  long long ld;
  const float* bi;           // [H]
  const float* bf;           // [H]
  const float* norm;         // [H DV]
  float* S;                  // [slots, H, D, DV]
  float* n;                  // [slots, H, D]
  float* m;                  // [slots, H]
  const int* cu_q;           // [B + 1] or null (decode)
  const int* context_lens;   // [B]
  const int* slots;          // [T] (decode)
  float* o;                  // [T, H, DV]: read-out before its norm
  float* n_new;              // [B, H, D]
  float* m_new;              // [B, H]
  void* out;                 // [T, H DV]
  int T, B, H, D, DV;
  float cap, eps, q_scale;
  __host__ __device__ int col_k() const { return H * D; }
  __host__ __device__ int col_v() const { return 2 * H * D; }
  __host__ __device__ int col_z() const { return 2 * H * D + H * DV; }
  __host__ __device__ int col_i() const { return 2 * H * (D + DV); }
};

constexpr int kCols = 32, kGroups = 8, kScan = kCols * kGroups;
constexpr int kMaxD = 512;

// R rows of one column per thread: rows group + 8 i
template <typename T, int R>
__global__ void __launch_bounds__(kScan) scan_kernel(const Args a) {
  __shared__ float sk[2][kMaxD], sq[2][kMaxD], sv[2][kCols], sg[2][2];
  __shared__ float red[kGroups][kCols], red_n[kGroups];
  const int b = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * kCols;
  const int r0 = a.cu_q[b], rows = a.cu_q[b + 1] - r0;
  if (rows <= 0) return;
  const int start = a.context_lens[b] - rows;
  const int D = a.D, DV = a.DV, H = a.H;
  const int tid = threadIdx.x, col = tid % kCols, grp = tid / kCols, c = c0 + col;
  const long long head = (long long)b * H + h;
  float s[R], n[2];
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int r = grp + kGroups * i;
    s[i] = (start > 0 && r < D && c < DV) ? a.S[(head * D + r) * DV + c] : 0.f;
  }
#pragma unroll
  for (int j = 0; j < 2; ++j) {
    const int r = tid + j * kScan;
    n[j] = (start > 0 && r < D) ? a.n[head * D + r] : 0.f;
  }
  float m = start > 0 ? a.m[head] : 0.f;
  const T* base = reinterpret_cast<const T*>(a.proj) + (long long)r0 * a.ld;
  const float bi = a.bi[h], bf = a.bf[h];
  auto fetch = [&](int t, int stage) {
    const T* row = base + (long long)t * a.ld;
    for (int r = tid; r < D; r += kScan) {
      sq[stage][r] = ld(row + h * D + r) * a.q_scale;
      sk[stage][r] = ld(row + a.col_k() + h * D + r);
    }
    if (tid < kCols) sv[stage][tid] = c0 + tid < DV ? ld(row + a.col_v() + h * DV + c0 + tid) : 0.f;
    if (tid == kCols) sg[stage][0] = input_gate(ld(row + a.col_i() + h) + bi, a.cap);
    if (tid == kCols + 32) sg[stage][1] = forget_gate(ld(row + a.col_i() + H + h) + bf, a.cap);
  };
  fetch(0, 0);
  __syncthreads();
  for (int t = 0; t < rows; ++t) {
    const int st_ = t & 1;
    const float i = sg[st_][0], f = sg[st_][1];
    const float m2 = fmaxf(f + m, i);
    const float keep = expf(f + m - m2), put = expf(i - m2);
    m = m2;
    const float v = put * sv[st_][col];
    float acc = 0.f;
#pragma unroll
    for (int j = 0; j < R; ++j) {
      const int r = grp + kGroups * j;
      if (r < D) {
        s[j] = fmaf(keep, s[j], sk[st_][r] * v);
        acc = fmaf(s[j], sq[st_][r], acc);
      }
    }
    float nq = 0.f;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int r = tid + j * kScan;
      if (r < D) {
        n[j] = fmaf(keep, n[j], put * sk[st_][r]);
        nq = fmaf(n[j], sq[st_][r], nq);
      }
    }
    nq = warp_sum(nq);
    red[grp][col] = acc;
    if (col == 0) red_n[grp] = nq;
    if (t + 1 < rows) fetch(t + 1, st_ ^ 1);
    __syncthreads();
    if (grp == 0 && c < DV) {
      float o = 0.f, d = 0.f;
#pragma unroll
      for (int g = 0; g < kGroups; ++g) { o += red[g][col]; d += red_n[g]; }
      a.o[((long long)(r0 + t) * H + h) * DV + c] = o / (fmaxf(fabsf(d), expf(-m)) + 1e-6f);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int r = grp + kGroups * i;
    if (r < D && c < DV) a.S[(head * D + r) * DV + c] = s[i];
  }
  if (blockIdx.x == 0) {
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int r = tid + j * kScan;
      if (r < D) a.n_new[head * D + r] = n[j];
    }
    if (tid == 0) a.m_new[head] = m;
  }
}

// a warp per (row, head); the CTAs behind those carry n and m over
template <typename T>
__global__ void __launch_bounds__(128) finish_kernel(const Args a) {
  const int lane = threadIdx.x & 31;
  const long long rows = (long long)a.T * a.H;
  const long long i = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  const int D = a.D, DV = a.DV, H = a.H;
  if (i >= rows) {
    const long long head = i - rows;
    if (head >= (long long)a.B * H) return;
    const int b = (int)(head / H);
    if (a.cu_q[b + 1] <= a.cu_q[b]) return;
    for (int r = lane; r < D; r += 32) a.n[head * D + r] = a.n_new[head * D + r];
    if (lane == 0) a.m[head] = a.m_new[head];
    return;
  }
  const long long t = i / H;
  const int h = (int)(i % H);
  const float* o = a.o + i * DV;
  float ss = 0.f;
  for (int c = lane; c < DV; c += 32) ss = fmaf(o[c], o[c], ss);
  const float rstd = 1.f / sqrtf(warp_sum(ss) / DV + a.eps);
  const T* z = reinterpret_cast<const T*>(a.proj) + t * a.ld + a.col_z() + h * DV;
  T* out = reinterpret_cast<T*>(a.out) + t * H * DV + h * DV;
  for (int c = lane; c < DV; c += 32) st(out + c, o[c] * rstd * a.norm[h * DV + c] / (1.f + expf(-ld(z + c))));
}

constexpr int kDec = 256;

// CTA (head, slot). VEC columns per thread; the threads of a column block share the rows.
template <typename T, int VEC>
__global__ void __launch_bounds__(kDec) decode_kernel(const Args a) {
  extern __shared__ float sh[];                    // k [D], q [D], o [DV], partial sums [kDec * VEC]
  __shared__ float red[kDec / 32];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int D = a.D, DV = a.DV, H = a.H;
  T* out = reinterpret_cast<T*>(a.out) + (long long)b * H * DV + h * DV;
  if (a.slots[b] < 0) {
    for (int c = tid; c < DV; c += kDec) st(out + c, 0.f);
    return;
  }
  const bool fresh = a.context_lens[b] <= 1;
  const long long head = (long long)b * H + h;
  const T* row = reinterpret_cast<const T*>(a.proj) + b * a.ld;
  float* k = sh;
  float* q = k + D;
  float* o = q + D;
  float* part = o + DV;
  const float i = input_gate(ld(row + a.col_i() + h) + a.bi[h], a.cap);
  const float f = forget_gate(ld(row + a.col_i() + H + h) + a.bf[h], a.cap);
  const float m0 = fresh ? 0.f : a.m[head];
  const float m = fmaxf(f + m0, i);
  const float keep = expf(f + m0 - m), put = expf(i - m);
  float nq = 0.f;
  for (int r = tid; r < D; r += kDec) {
    const float kk = put * ld(row + a.col_k() + h * D + r), qq = ld(row + h * D + r) * a.q_scale;
    const float n = fmaf(keep, fresh ? 0.f : a.n[head * D + r], kk);
    a.n[head * D + r] = n;
    nq = fmaf(n, qq, nq);
    k[r] = kk;
    q[r] = qq;
  }
  nq = warp_sum(nq);
  if ((tid & 31) == 0) red[tid >> 5] = nq;
  __syncthreads();                                 // every thread has read m
  if (tid == 0) a.m[head] = m;
  nq = 0.f;
#pragma unroll
  for (int w = 0; w < kDec / 32; ++w) nq += red[w];
  const float inv = 1.f / (fmaxf(fabsf(nq), expf(-m)) + 1e-6f);
  const int nv = DV / VEC, cols = nv < kDec ? nv : kDec, groups = kDec / cols;
  const int grp = tid / cols, ci = tid % cols;
  const bool on = grp < groups;
  for (int c0 = 0; c0 < nv; c0 += cols) {
    const int cv = c0 + ci;
    float acc[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
    if (on && cv < nv) {
      float v[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] = ld(row + a.col_v() + h * DV + cv * VEC + e);
      float* s = a.S + head * D * DV + (long long)cv * VEC;
#pragma unroll 4
      for (int r = grp; r < D; r += groups) {
        float x[VEC];
        if (fresh) {
#pragma unroll
          for (int e = 0; e < VEC; ++e) x[e] = k[r] * v[e];
        } else if constexpr (VEC == 4) {
          const float4 y = *reinterpret_cast<const float4*>(s + (long long)r * DV);
          x[0] = fmaf(keep, y.x, k[r] * v[0]); x[1] = fmaf(keep, y.y, k[r] * v[1]);
          x[2] = fmaf(keep, y.z, k[r] * v[2]); x[3] = fmaf(keep, y.w, k[r] * v[3]);
        } else {
          x[0] = fmaf(keep, s[(long long)r * DV], k[r] * v[0]);
        }
        if constexpr (VEC == 4) *reinterpret_cast<float4*>(s + (long long)r * DV) = make_float4(x[0], x[1], x[2], x[3]);
        else s[(long long)r * DV] = x[0];
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc[e] = fmaf(x[e], q[r], acc[e]);
      }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) part[tid * VEC + e] = acc[e];
    __syncthreads();
    if (grp == 0 && cv < nv) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        float x = 0.f;
        for (int g = 0; g < groups; ++g) x += part[(g * cols + ci) * VEC + e];
        o[cv * VEC + e] = x * inv;
      }
    }
    __syncthreads();
  }
  float ss = 0.f;
  for (int c = tid; c < DV; c += kDec) ss = fmaf(o[c], o[c], ss);
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int w = 0; w < kDec / 32; ++w) ss += red[w];
  const float rstd = 1.f / sqrtf(ss / DV + a.eps);
  const T* z = row + a.col_z() + h * DV;
  for (int c = tid; c < DV; c += kDec) st(out + c, o[c] * rstd * a.norm[h * DV + c] / (1.f + expf(-ld(z + c))));
}

template <typename T>
int portions(const Args& a, cudaStream_t stream) {
  const dim3 grid((a.DV + kCols - 1) / kCols, a.H, a.B);
  const int r = (a.D + kGroups - 1) / kGroups;
  if (r <= 8) scan_kernel<T, 8><<<grid, kScan, 0, stream>>>(a);
  else if (r <= 16) scan_kernel<T, 16><<<grid, kScan, 0, stream>>>(a);
  else if (r <= 32) scan_kernel<T, 32><<<grid, kScan, 0, stream>>>(a);
  else scan_kernel<T, 64><<<grid, kScan, 0, stream>>>(a);
  const long long items = (long long)a.T * a.H + (long long)a.B * a.H;
  finish_kernel<T><<<(unsigned)((items + 3) / 4), 128, 0, stream>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : 2;
}

template <typename T>
int decode(const Args& a, cudaStream_t stream) {
  const bool vec = a.DV % 4 == 0;
  const size_t smem = (size_t)(2 * a.D + a.DV + kDec * (vec ? 4 : 1)) * sizeof(float);
  if (smem > 48 * 1024) { mfb_host::set_error("matrix_memory: D=%d DV=%d", a.D, a.DV); return 1; }
  const dim3 grid(a.H, a.B);
  if (vec) decode_kernel<T, 4><<<grid, kDec, smem, stream>>>(a);
  else decode_kernel<T, 1><<<grid, kDec, smem, stream>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : 2;
}

}  // namespace mmem
}  // namespace mfb

extern "C" {
using namespace mfb;

// fp32 values of scratch for portions.
long long mfb_matrix_memory_scratch_floats(int T, int B, int H, int D, int DV) {
  return (long long)T * H * DV + (long long)B * H * (D + 1);
}

// See the head of this file. cu_q [B + 1] (device): portions, with scratch; null: one row per slot (T == B). longest: rows of the
// longest portion. Key sizes up to 512, value sizes up to 4096. f32 = 1: activations are fp32, else bf16.
int mfb_matrix_memory(const void* proj, long long ld, const float* bi, const float* bf, const float* norm, float* S, float* n,
                      float* m, const int* cu_q, const int* context_lens, const int* slots, float* scratch, void* out, int T, int B,
                      int H, int D, int DV, int longest, float cap, float eps, int f32, cudaStream_t stream) {
  if (T <= 0 || B <= 0) return 0;
  if (H < 1 || D < 1 || DV < 1 || D > mmem::kMaxD || DV > 4096 || H > 65535 || B > 65535 || ld < 2LL * H * (D + DV) + 2 * H ||
      (!cu_q && T != B) || (cu_q && !scratch)) {
    mfb_host::set_error("matrix_memory: T=%d B=%d H=%d D=%d DV=%d ld=%lld", T, B, H, D, DV, ld);
    return 1;
  }
  (void)longest;
  mmem::Args a;
  a.proj = proj; a.ld = ld; a.bi = bi; a.bf = bf; a.norm = norm; a.S = S; a.n = n; a.m = m; a.cu_q = cu_q;
  a.context_lens = context_lens; a.slots = slots; a.out = out;
  a.o = scratch; a.n_new = scratch + (long long)T * H * DV; a.m_new = a.n_new + (long long)B * H * D;
  a.T = T; a.B = B; a.H = H; a.D = D; a.DV = DV; a.cap = cap; a.eps = eps; a.q_scale = 1.f / sqrtf((float)D);
  int rc;
  if (cu_q) rc = f32 ? mmem::portions<float>(a, stream) : mmem::portions<__nv_bfloat16>(a, stream);
  else rc = f32 ? mmem::decode<float>(a, stream) : mmem::decode<__nv_bfloat16>(a, stream);
  if (rc == 2) mfb_host::set_error("matrix_memory: launch failed");
  return rc;
}

}  // extern "C"
