// State-space mixer with a scalar decay per head (the recurrence of Mamba-2) over ragged batches (sm_100a, bf16 or fp32
// activations).
//
// A row of the projection holds z [H P] | x [H P] | B [G N] | C [G N] | dt [H]. x, B and C pass a causal convolution per channel
// with a bias, and silu. With dt = softplus(dt + dt_bias) and head h in group h / (H / G):
//   S' = e^(-e^A_h dt) S + dt B x^T,   y = S'^T C + D_h x          S [N, P]
// and the result is RMS-normed in `norm_groups` parts of y * silu(z), times `norm`. S [slots, H, N, P] is fp32; the last inputs of
// the convolution are kept in a ring [slots, taps, H P + 2 G N], the input at position p in place p % taps: one place more than a
// token reads, so that a decode step may write its own while others read. Row b of a batch uses slot b. A sequence that starts at
// position 0 reads neither, so a slot changes hands without being cleared.
//
//   conv_kernel:             convolution and silu of portions, a run of rows per thread
//   gates_kernel, chunk_kernel: portions of 16-bit models in chunks of 64 tokens on the tensor cores (see there)
//   scan_kernel:             portions of 32-bit models and of other sizes, token by token on the FMA pipes
//   decode_kernel:           one row per slot: convolution, recurrence, gate
//   finish_kernel:           norm of the gated read-out in place; for portions also the ring
#include "mma_sync.cuh"

namespace mfb {
namespace ssm {

__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
template <typename T>
__device__ __forceinline__ float silu(float z) {
  if constexpr (sizeof(T) == 2) return __fdividef(z, 1.f + __expf(-fmaxf(z, -80.f)));      // the quotient's divisor stays in reach
  else return z / (1.f + expf(-z));
}
template <int VEC>
__device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[VEC]) {
  if constexpr (VEC == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
    const float2 g = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    v[0] = f.x; v[1] = f.y; v[2] = g.x; v[3] = g.y;
  } else if constexpr (VEC == 8) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) { const float2 f = __bfloat1622float2(h[i]); v[2 * i] = f.x; v[2 * i + 1] = f.y; }
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = ld(p + i);
  }
}
template <int VEC>
__device__ __forceinline__ void load(const float* p, float (&v)[VEC]) {
  if constexpr (VEC % 4 == 0) {
#pragma unroll
    for (int i = 0; i < VEC; i += 4) {
      const float4 a = *reinterpret_cast<const float4*>(p + i);
      v[i] = a.x; v[i + 1] = a.y; v[i + 2] = a.z; v[i + 3] = a.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = p[i];
  }
}
template <int VEC>
__device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[VEC]) {
  if constexpr (VEC == 4) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
  } else if constexpr (VEC == 8) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]),
                                              pack_bf16x2(v[6], v[7]));
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) st(p + i, v[i]);
  }
}
template <int VEC>
__device__ __forceinline__ void store(float* p, const float (&v)[VEC]) {
  if constexpr (VEC % 4 == 0) {
#pragma unroll
    for (int i = 0; i < VEC; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) p[i] = v[i];
  }
}

// One step of a decay e^a, a <= 0, as s <- most * s + rest * s: with (1, e^a - 1) where the decay is slow, so that the rounding of
// a factor close to one does not add up over the thousands of tokens that such a state remembers, else with (0, e^a).
struct Decay {
  float most, rest;
  __device__ __forceinline__ explicit Decay(float a) {
    const bool slow = a > -0.5f;
    most = slow ? 1.f : 0.f;
    rest = slow ? expm1f(a) : expf(a);
  }
  __device__ __forceinline__ float operator()(float s, float add) const { return fmaf(rest, s, fmaf(most, s, add)); }
};

struct Args {
  const void* proj;          // [T, >= 2 H P + 2 G N + H]
  long long ld;
  const float* conv;         // [taps, C]; the last row belongs to the current token
  const float* conv_b;       // [C]
  const float* dt_bias;      // [H]
  const float* a_log;        // [H]
  const float* d;            // [H]
  const float* norm;         // [H P]
  void* ring;                // [slots, taps, C]
  float* S;                  // [slots, H, N, P]
  const int* cu_q;           // [B + 1] or null (decode)
  const int* context_lens;   // [B]
  const int* slots;          // [T] (decode)
  float4* gates;             // [H, T] of the chunks: log decay up to the token (high, low), dt
  void* xbc;                 // [T, C], rows ld_x apart: after convolution and silu
  long long ld_x;
  void* out;                 // [T, H P]
  int T, B, H, P, N, G, taps, norm_groups;
  int rows;                  // rows (convolution) or heads (decode) per CTA
  float eps;
  __host__ __device__ int inner() const { return H * P; }
  __host__ __device__ int channels() const { return H * P + 2 * G * N; }
  __host__ __device__ int col_dt() const { return 2 * H * P + 2 * G * N; }
};

constexpr int kMaxTaps = 16, kAhead = 4;

// VEC channels per thread, a.rows rows per CTA; TM: bound of the taps (weights are padded with zeros in front)
template <typename T, int VEC, int TM>
__global__ void __launch_bounds__(128) conv_kernel(const Args a) {
  const int C = a.channels(), c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  if (c >= C) return;
  const int r0 = blockIdx.x * a.rows, r1 = min(r0 + a.rows, a.T);
  int lo = 0, hi = a.B - 1;                  // last sequence that starts at or before the first row (and is not empty there)
  while (lo < hi) {
    const int mid = (lo + hi + 1) / 2;
    if (a.cu_q[mid] <= r0) lo = mid; else hi = mid - 1;
  }
  int b = lo;
  const int skip = TM - a.taps;
  float w[TM][VEC], bias[VEC], win[TM][VEC];
#pragma unroll
  for (int j = 0; j < TM; ++j) {
    if (j >= skip) load<VEC>(a.conv + (long long)(j - skip) * C + c, w[j]);
    else {
#pragma unroll
      for (int i = 0; i < VEC; ++i) w[j][i] = 0.f;
    }
  }
  load<VEC>(a.conv_b + c, bias);
  const T* src = reinterpret_cast<const T*>(a.proj) + a.inner() + c;
  auto restart = [&](int r) {                // inputs in front of row r of sequence b
    const int q0 = a.cu_q[b], start = a.context_lens[b] - (a.cu_q[b + 1] - q0);
    const T* ring = reinterpret_cast<const T*>(a.ring) + (long long)b * a.taps * C + c;
#pragma unroll
    for (int j = 0; j + 1 < TM; ++j) {
      const int back = TM - 1 - j;           // tokens before row r
      const int at = r - back, p = start + at - q0;
      if (back >= a.taps || p < 0) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) win[j][i] = 0.f;
      } else if (at >= q0) load<VEC>(src + (long long)at * a.ld, win[j]);
      else load<VEC>(ring + (long long)(p % a.taps) * C, win[j]);
    }
  };
  restart(r0);
  int end = a.cu_q[b + 1];
  // kAhead rows are on their way at a time
  float next[kAhead][VEC];
  for (int r8 = r0; r8 < r1; r8 += kAhead) {
#pragma unroll
    for (int u = 0; u < kAhead; ++u)
      if (r8 + u < r1) load<VEC>(src + (long long)(r8 + u) * a.ld, next[u]);
#pragma unroll
    for (int u = 0; u < kAhead; ++u) {
      const int r = r8 + u;
      if (r >= r1) break;
      if (r >= end) {
        while (r >= a.cu_q[b + 1]) ++b;
        end = a.cu_q[b + 1];
        restart(r);
      }
#pragma unroll
      for (int i = 0; i < VEC; ++i) win[TM - 1][i] = next[u][i];
      float y[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        y[i] = bias[i];
#pragma unroll
        for (int j = 0; j < TM; ++j) y[i] = fmaf(w[j][i], win[j][i], y[i]);
        y[i] = silu<T>(y[i]);
      }
      store<VEC>(reinterpret_cast<T*>(a.xbc) + (long long)r * a.ld_x + c, y);
#pragma unroll
      for (int j = 0; j + 1 < TM; ++j)
#pragma unroll
        for (int i = 0; i < VEC; ++i) win[j][i] = win[j + 1][i];
    }
  }
}

constexpr int kCols = 32, kGroups = 8, kScan = kCols * kGroups;
constexpr int kMaxN = 512;

// 32 columns of one head's S per CTA; R rows of one column per thread: rows group + 8 i
template <typename T, int R>
__global__ void __launch_bounds__(kScan) scan_kernel(const Args a) {
  __shared__ float sb[2][kMaxN], sc[2][kMaxN], sx[2][kCols], sdt[2];
  __shared__ float red[kGroups][kCols];
  const int b = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * kCols;
  const int r0 = a.cu_q[b], rows = a.cu_q[b + 1] - r0;
  if (rows <= 0) return;
  const int start = a.context_lens[b] - rows;
  const int N = a.N, P = a.P, H = a.H, inner = a.inner(), g = h / (H / a.G);
  const int tid = threadIdx.x, col = tid % kCols, grp = tid / kCols, c = c0 + col;
  const long long head = (long long)b * H + h;
  float s[R];
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int r = grp + kGroups * i;
    s[i] = (start > 0 && r < N && c < P) ? a.S[(head * N + r) * P + c] : 0.f;
  }
  const T* xbc = reinterpret_cast<const T*>(a.xbc) + (long long)r0 * a.ld_x;
  const T* proj = reinterpret_cast<const T*>(a.proj) + (long long)r0 * a.ld;
  const float rate = -expf(a.a_log[h]), bias = a.dt_bias[h], d = a.d[h];
  auto fetch = [&](int t, int stage) {
    const T* row = xbc + (long long)t * a.ld_x;
    for (int r = tid; r < N; r += kScan) {
      sb[stage][r] = ld(row + inner + g * N + r);
      sc[stage][r] = ld(row + inner + (a.G + g) * N + r);
    }
    if (tid < kCols) sx[stage][tid] = c0 + tid < P ? ld(row + h * P + c0 + tid) : 0.f;
    if (tid == kCols) sdt[stage] = softplus(ld(proj + (long long)t * a.ld + a.col_dt() + h) + bias);
  };
  fetch(0, 0);
  __syncthreads();
  for (int t = 0; t < rows; ++t) {
    const int stage = t & 1;
    const float dt = sdt[stage], x = sx[stage][col];
    const Decay decay(rate * dt);
    const float v = dt * x;
    float acc = 0.f;
#pragma unroll
    for (int j = 0; j < R; ++j) {
      const int r = grp + kGroups * j;
      if (r < N) {
        s[j] = decay(s[j], sb[stage][r] * v);
        acc = fmaf(s[j], sc[stage][r], acc);
      }
    }
    red[grp][col] = acc;
    if (t + 1 < rows) fetch(t + 1, stage ^ 1);
    __syncthreads();
    if (grp == 0 && c < P) {
      float y = d * x;
#pragma unroll
      for (int k = 0; k < kGroups; ++k) y += red[k][col];
      const float z = ld(proj + (long long)t * a.ld + h * P + c);
      st(reinterpret_cast<T*>(a.out) + (long long)(r0 + t) * inner + h * P + c, y * silu<T>(z));
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int r = grp + kGroups * i;
    if (r < N && c < P) a.S[(head * N + r) * P + c] = s[i];
  }
}

constexpr int kDec = 256;

// CTA (a.rows heads of a group, slot): B and C once for its heads. VEC columns per thread; the threads of a column block share the
// rows of S.
template <typename T, int VEC>
__global__ void __launch_bounds__(kDec) decode_kernel(const Args a) {
  extern __shared__ float sh[];                    // B [N], C [N], x [heads P], partial sums [heads][kDec * VEC]
  const int heads = a.rows, h0 = blockIdx.x * heads, b = blockIdx.y, tid = threadIdx.x;
  const int N = a.N, P = a.P, H = a.H, inner = a.inner(), C = a.channels(), per = H / a.G, g = h0 / per, cols_x = heads * P;
  T* out = reinterpret_cast<T*>(a.out) + (long long)b * inner + h0 * P;
  if (a.slots[b] < 0) {
    for (int c = tid; c < cols_x; c += kDec) st(out + c, 0.f);
    return;
  }
  const int pos = a.context_lens[b] - 1;
  const bool fresh = pos <= 0;
  const T* row = reinterpret_cast<const T*>(a.proj) + b * a.ld;
  T* ring = reinterpret_cast<T*>(a.ring) + (long long)b * a.taps * C;
  float* part = sh + 2 * N + cols_x;
  const int place = pos % a.taps;
  for (int i = tid; i < 2 * N + cols_x; i += kDec) {
    const int c = i < N ? inner + g * N + i : i < 2 * N ? inner + a.G * N + g * N + i - N : h0 * P + i - 2 * N;
    const float now = ld(row + inner + c);
    float y = fmaf(a.conv[(long long)(a.taps - 1) * C + c], now, a.conv_b[c]);
    for (int j = 1; j < a.taps && j <= pos; ++j) {
      const int at = place >= j ? place - j : place - j + a.taps;
      y = fmaf(a.conv[(long long)(a.taps - 1 - j) * C + c], ld(ring + (long long)at * C + c), y);
    }
    // the channels of a group's B and C are written by its first heads
    if (i >= 2 * N || h0 == g * per) st(ring + (long long)place * C + c, now);
    y = silu<T>(y);
    // what enters the recurrence after the convolution is an activation
    if constexpr (sizeof(T) == 2) y = __bfloat162float(__float2bfloat16_rn(y));
    sh[i] = y;
  }
  __syncthreads();
  const float* sB = sh;
  const float* sC = sh + N;
  const float* sX = sh + 2 * N;
  const int nv = P / VEC, cols = nv < kDec ? nv : kDec, groups = kDec / cols;
  const int grp = tid / cols, ci = tid % cols;
  const bool on = grp < groups;
  for (int c0 = 0; c0 < nv; c0 += cols) {
    const int cv = c0 + ci;
    for (int k = 0; k < heads; ++k) {
      const int h = h0 + k;
      float acc[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
      if (on && cv < nv) {
        const float dt = softplus(ld(row + a.col_dt() + h) + a.dt_bias[h]);
        const Decay decay(-expf(a.a_log[h]) * dt);
        float v[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] = dt * sX[k * P + cv * VEC + e];
        float* s = a.S + ((long long)b * H + h) * N * P + (long long)cv * VEC;
#pragma unroll 8
        for (int r = grp; r < N; r += groups) {
          float x[VEC];
          if (fresh) {
#pragma unroll
            for (int e = 0; e < VEC; ++e) x[e] = 0.f;
          } else load<VEC>(s + (long long)r * P, x);
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            x[e] = decay(x[e], sB[r] * v[e]);
            acc[e] = fmaf(x[e], sC[r], acc[e]);
          }
          store<VEC>(s + (long long)r * P, x);
        }
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) part[(k * kDec + tid) * VEC + e] = acc[e];
    }
    __syncthreads();
    const int width = min(cols * VEC, P - c0 * VEC);
    for (int i = tid; i < heads * width; i += kDec) {
      const int k = i / width, c = i % width, col = k * P + c0 * VEC + c;
      float y = a.d[h0 + k] * sX[col];
      for (int j = 0; j < groups; ++j) y += part[k * kDec * VEC + j * cols * VEC + c];
      st(out + col, y * silu<T>(ld(row + h0 * P + col)));
    }
    __syncthreads();
  }
}

// RMS norm in place: blockDim.x threads per (row, part), K accesses of VEC columns each; a warp each where blockDim.y > 1. The
// CTAs behind those move a sequence's last inputs of the convolution into its ring.
constexpr int kRingCols = 512;
template <typename T, int VEC, int K>
__global__ void __launch_bounds__(1024) finish_kernel(const Args a) {
  __shared__ float red[32];
  const unsigned items = (unsigned)(a.T * a.norm_groups), ctas = (items + blockDim.y - 1) / blockDim.y;
  const int inner = a.inner();
  if (blockIdx.x >= ctas) {                           // a CTA per sequence, token and kRingCols channels
    const int C = a.channels(), slices = (C + kRingCols - 1) / kRingCols;
    const int i = (int)(blockIdx.x - ctas), c0 = i % slices * kRingCols, j = i / slices % a.taps, b = i / slices / a.taps;
    if (j >= a.cu_q[b + 1] - a.cu_q[b]) return;
    const T* src = reinterpret_cast<const T*>(a.proj) + (long long)(a.cu_q[b + 1] - 1 - j) * a.ld + inner;
    T* dst = reinterpret_cast<T*>(a.ring) + ((long long)b * a.taps + (a.context_lens[b] - 1 - j) % a.taps) * C;
    for (int c = c0 + threadIdx.y * blockDim.x + threadIdx.x; c < min(C, c0 + kRingCols); c += blockDim.x * blockDim.y) dst[c] = src[c];
    return;
  }
  const int gw = inner / a.norm_groups, nvec = gw / VEC;
  const unsigned item = blockIdx.x * blockDim.y + threadIdx.y;
  if (item >= items) return;
  const unsigned t = item / a.norm_groups;
  const int c0 = (int)(item % a.norm_groups) * gw;
  T* row = reinterpret_cast<T*>(a.out) + (long long)t * inner + c0;
  float v[K][VEC], ss = 0.f;
#pragma unroll
  for (int k = 0; k < K; ++k) {
    const int c = threadIdx.x + k * blockDim.x;
    if (c < nvec) {
      load<VEC>(row + c * VEC, v[k]);
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss = fmaf(v[k][i], v[k][i], ss);
    }
  }
  ss = warp_sum(ss);
  if (blockDim.x > 32) {
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.f;
    for (int w = 0; w < (int)(blockDim.x >> 5); ++w) ss += red[w];
  }
  const float rstd = inv_sqrt(ss / gw + a.eps);
#pragma unroll
  for (int k = 0; k < K; ++k) {
    const int c = threadIdx.x + k * blockDim.x;
    if (c < nvec) {
      float w[VEC];
      load<VEC>(a.norm + c0 + c * VEC, w);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[k][i] *= rstd * w[i];
      store<VEC>(row + c * VEC, v[k]);
    }
  }
}

// ---- portions in chunks of 64 tokens ----------------------------------------------------------------------------------------
// With b_t the sum of the log decays of a chunk up to token t (so e^b_t <= 1 and it falls):
//   y_t = e^b_t S^T C_t + sum_{s <= t} (C_t . B_s) e^(b_t - b_s) dt_s x_s + D x_t
//   after the last token: S <- e^b S + sum_s B_s (e^(b - b_s) dt_s x_s)^T
// The sums do not depend on what came before the chunk: gates_kernel works them out for all chunks at once, in fp64, as pairs of
// fp32 numbers (their differences stay exact where the sums are large). chunk_kernel walks over the chunks of one head: four warps
// hold 16 columns of S each, transposed, as fp32 MMA accumulators. x, B and C enter the products as they are (bf16); fp32 factors
// enter as sums of bf16 numbers: two for S and the weights in the read-out, three for the weighted x that go into S, whose error
// would stay.
constexpr int kChunk = 64;

// a warp per head, two tokens per lane
constexpr int kGateHeads = 8;
template <typename T>
__global__ void __launch_bounds__(32 * kGateHeads) gates_kernel(const Args a) {
  __shared__ float sh[kChunk][kGateHeads + 1];       // raw step sizes
  const int b = blockIdx.y, r0 = a.cu_q[b], rows = a.cu_q[b + 1] - r0, t0 = blockIdx.x * kChunk, h0 = blockIdx.z * kGateHeads;
  if (t0 >= rows) return;
  const int n = min(kChunk, rows - t0), heads = min(kGateHeads, a.H - h0);
  for (int i = threadIdx.x; i < n * kGateHeads; i += blockDim.x) {
    const int t = i / kGateHeads, k = i % kGateHeads;
    if (k < heads) sh[t][k] = ld(reinterpret_cast<const T*>(a.proj) + (long long)(r0 + t0 + t) * a.ld + a.col_dt() + h0 + k);
  }
  __syncthreads();
  const int lane = threadIdx.x & 31, own = threadIdx.x >> 5;
  if (own < heads) {
    const int h = h0 + own;
    const float rate = -expf(a.a_log[h]), bias = a.dt_bias[h];
    float dt[2];
    double f[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = 2 * lane + e;
      dt[e] = t < n ? softplus(sh[t][own] + bias) : 0.f;
      f[e] = (double)rate * (double)dt[e];
    }
    double sum = f[0] + f[1];
#pragma unroll
    for (int o = 1; o < 32; o *= 2) {
      const double up = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += up;
    }
    float4* g = a.gates + (long long)h * a.T + r0 + t0 + 2 * lane;
    auto put = [](float4* p, double x, float dt_) {
      const float hi = static_cast<float>(x);
      *p = make_float4(hi, static_cast<float>(x - hi), dt_, 0.f);
    };
    if (2 * lane < n) put(g, sum - f[1], dt[0]);
    if (2 * lane + 1 < n) put(g + 1, sum, dt[1]);
  }
}

// NP: padded state size; STAGES: buffers of C, B and x
template <int NP, int STAGES>
struct ChunkShape {
  static constexpr int kCPitch = NP * 2 + 16, kXPitch = 64 * 2 + 16;      // bytes; rows shift by a bank group
  static constexpr int kCBytes = kChunk * kCPitch, kXBytes = kChunk * kXPitch;
  static constexpr int kStage = 2 * kCBytes + kXBytes + kChunk * 16;
  static constexpr int kSmem = STAGES * kStage + 2 * kXBytes + 2 * kChunk * 4;
};

template <int NP, int STAGES>
__global__ void __launch_bounds__(128, 2) chunk_kernel(const Args p) {
  using Sh = ChunkShape<NP, STAGES>;
  constexpr int KS = NP / 16, NT = NP / 8;
  extern __shared__ __align__(16) uint8_t smem[];
  const int b = blockIdx.z, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int r0 = p.cu_q[b], rows = p.cu_q[b + 1] - r0;
  if (rows <= 0) return;
  const int start = p.context_lens[b] - rows, N = p.N, P = p.P, H = p.H, inner = p.inner(), group = h / (H / p.G);
  const int slice = blockIdx.x * 64, v0 = slice + warp * 16;
  const int g = lane >> 2, tq = lane & 3;
  uint8_t* sP = smem + STAGES * Sh::kStage;           // weights: high, low
  float* sScale = reinterpret_cast<float*>(sP + 2 * Sh::kXBytes);     // e^b_t
  float* sW = sScale + kChunk;                        // weight of a token in the state after the chunk
  const long long head = (long long)b * H + h;
  const __nv_bfloat16* base = reinterpret_cast<const __nv_bfloat16*>(p.xbc) + (long long)r0 * p.ld_x;
  const __nv_bfloat16* zbase = reinterpret_cast<const __nv_bfloat16*>(p.proj) + (long long)r0 * p.ld + h * P;
  __nv_bfloat16* obase = reinterpret_cast<__nv_bfloat16*>(p.out) + (long long)r0 * inner + h * P;
  const float skip = p.d[h];

  float s[NT][4];                                     // S^T: rows v0 + g, v0 + g + 8; columns 8 j + 2 tq, + 1
  {
    const float* S = p.S + head * N * P;
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = 8 * j + 2 * tq + (e & 1), v = v0 + g + (e >> 1) * 8;
        s[j][e] = (start > 0 && d < N && v < P) ? S[(long long)d * P + v] : 0.f;
      }
  }

  const int chunks = (rows + kChunk - 1) / kChunk;
  auto fetch = [&](int c) {
    uint8_t* st = smem + (c % STAGES) * Sh::kStage;
    const uint32_t sc = smem_u32(st);
    const int n = min(kChunk, rows - c * kChunk);
    for (int i = tid; i < kChunk * (NP / 8); i += 128) {
      const int t = i / (NP / 8), d = (i % (NP / 8)) * 8;
      const bool in = t < n && d < N;
      const __nv_bfloat16* src = base + (long long)(c * kChunk + (in ? t : 0)) * p.ld_x + inner + group * N + (in ? d : 0);
      cp16(sc + t * Sh::kCPitch + d * 2, src + p.G * N, in ? 16 : 0);
      cp16(sc + Sh::kCBytes + t * Sh::kCPitch + d * 2, src, in ? 16 : 0);
    }
    for (int i = tid; i < kChunk * 8; i += 128) {
      const int t = i / 8, v = (i % 8) * 8;
      const bool in = t < n && slice + v < P;
      const __nv_bfloat16* src = base + (long long)(c * kChunk + (in ? t : 0)) * p.ld_x + h * P + (in ? slice + v : 0);
      cp16(sc + 2 * Sh::kCBytes + t * Sh::kXPitch + v * 2, src, in ? 16 : 0);
    }
    // padding tokens have step size zero
    const float4* gates = p.gates + (long long)h * p.T + r0 + c * kChunk;
    if (tid < kChunk) cp16(sc + 2 * Sh::kCBytes + Sh::kXBytes + tid * 16, gates + (tid < n ? tid : 0), tid < n ? 16 : 0);
    cp_commit();
  };
  fetch(0);
  for (int c = 0; c < chunks; ++c) {
    const int n = min(kChunk, rows - c * kChunk);
    if (STAGES > 1 && c + 1 < chunks) { fetch(c + 1); cp_wait<1>(); }
    else cp_wait<0>();
    __syncthreads();
    uint8_t* st = smem + (c % STAGES) * Sh::kStage;
    const uint32_t sc = smem_u32(st), sb = sc + Sh::kCBytes, sx = sb + Sh::kCBytes, sp = smem_u32(sP);
    const uint8_t* xt = st + 2 * Sh::kCBytes;
    const float4* sg = reinterpret_cast<const float4*>(xt + Sh::kXBytes);
    const float4 last_gate = sg[n - 1];
    const float keep = expf(last_gate.x + last_gate.y);
    if (tid < kChunk) {
      const float4 gt = sg[tid];
      sW[tid] = tid < n ? gt.z * expf((last_gate.x - gt.x) + (last_gate.y - gt.y)) : 0.f;
      sScale[tid] = expf(gt.x + gt.y);
    }
    // gates of the warp's 16 columns: rows m * 16 + g (+ 8), loaded ahead of the products
    uint32_t z[4][2][2];
    if (v0 < P) {
#pragma unroll
      for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int t = m * 16 + g + 8 * r;
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const int v = v0 + j * 8 + 2 * tq;
            z[m][r][j] = (t < n && v < P) ? *reinterpret_cast<const uint32_t*>(zbase + (long long)(c * kChunk + t) * p.ld + v) : 0u;
          }
        }
    }
    // ---- scores of the warp's 16 tokens and their weights ----
    {
      float acc[8][4] = {};
      const int last = 2 * warp + 1;                  // key tiles up to the diagonal
#pragma unroll
      for (int k = 0; k < KS; ++k) {
        uint32_t ca[4];
        ldsm4(ca, sc + (warp * 16 + (lane & 15)) * Sh::kCPitch + k * 32 + (lane >> 4) * 16);
#pragma unroll
        for (int j = 0; j < 8; j += 2)
          if (j <= last) {
            uint32_t bb[4];                           // tiles j and j + 1, both halves of the 16 dimensions
            ldsm4(bb, sb + (j * 8 + (lane & 7) + (lane >> 4) * 8) * Sh::kCPitch + k * 32 + ((lane >> 3) & 1) * 16);
            mma(acc[j], ca, bb[0], bb[1]);
            mma(acc[j + 1], ca, bb[2], bb[3]);
          }
      }
      float th[2], tl[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const float4 gt = sg[warp * 16 + g + 8 * r];
        th[r] = gt.x;
        tl[r] = gt.y;
      }
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (j <= last) {
          const int s0 = j * 8 + 2 * tq;
          const float4 g0 = sg[s0], g1 = sg[s0 + 1];
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            const int t = warp * 16 + g + 8 * r;
            const bool in = t < n;
            float w0 = in && s0 <= t ? acc[j][2 * r] * (g0.z * __expf((th[r] - g0.x) + (tl[r] - g0.y))) : 0.f;
            float w1 = in && s0 + 1 <= t ? acc[j][2 * r + 1] * (g1.z * __expf((th[r] - g1.x) + (tl[r] - g1.y))) : 0.f;
            uint8_t* dst = sP + t * Sh::kXPitch + s0 * 2;
            *reinterpret_cast<uint32_t*>(dst) = take_bf16(w0, w1);
            *reinterpret_cast<uint32_t*>(dst + Sh::kXBytes) = take_bf16(w0, w1);
          }
        }
    }
    __syncthreads();
    if (v0 < P) {
      // ---- read-out of the warp's 16 columns for all tokens ----
      float o[4][2][4] = {};
#pragma unroll
      for (int k = 0; k < KS; ++k) {
        uint32_t hi[4], lo[4];                        // S as a K x N operand: columns v0.. (0, 1), v0 + 8.. (2, 3)
#pragma unroll
        for (int e = 0; e < 2; ++e)
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            float x = s[2 * k + j][2 * e], y = s[2 * k + j][2 * e + 1];
            hi[2 * e + j] = take_bf16(x, y);
            lo[2 * e + j] = take_bf16(x, y);
          }
#pragma unroll
        for (int m = 0; m < 4; ++m) {
          uint32_t ca[4];
          ldsm4(ca, sc + (m * 16 + (lane & 15)) * Sh::kCPitch + k * 32 + (lane >> 4) * 16);
          mma(o[m][0], ca, hi[0], hi[1]);
          mma(o[m][1], ca, hi[2], hi[3]);
          mma(o[m][0], ca, lo[0], lo[1]);
          mma(o[m][1], ca, lo[2], lo[3]);
        }
      }
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        const float s0 = sScale[m * 16 + g], s1 = sScale[m * 16 + g + 8];
#pragma unroll
        for (int j = 0; j < 2; ++j) { o[m][j][0] *= s0; o[m][j][1] *= s0; o[m][j][2] *= s1; o[m][j][3] *= s1; }
      }
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        uint32_t xb[4];                               // tokens 16 k.. of columns v0.. (0, 1), v0 + 8.. (2, 3)
        ldsm4t(xb, sx + (k * 16 + (lane & 15)) * Sh::kXPitch + warp * 32 + (lane >> 4) * 16);
#pragma unroll
        for (int m = k; m < 4; ++m) {
          const uint32_t at = sp + (m * 16 + (lane & 15)) * Sh::kXPitch + k * 32 + (lane >> 4) * 16;
          uint32_t wa[4];
          ldsm4(wa, at);
          mma(o[m][0], wa, xb[0], xb[1]);
          mma(o[m][1], wa, xb[2], xb[3]);
          ldsm4(wa, at + Sh::kXBytes);
          mma(o[m][0], wa, xb[0], xb[1]);
          mma(o[m][1], wa, xb[2], xb[3]);
        }
      }
#pragma unroll
      for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int t = m * 16 + g + 8 * r;
          if (t >= n) continue;
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const int v = v0 + j * 8 + 2 * tq;
            if (v >= P) continue;
            const float2 x = __bfloat1622float2(
                *reinterpret_cast<const __nv_bfloat162*>(xt + t * Sh::kXPitch + (warp * 16 + j * 8 + 2 * tq) * 2));
            const float2 zz = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&z[m][r][j]));
            const float y0 = fmaf(skip, x.x, o[m][j][2 * r]), y1 = fmaf(skip, x.y, o[m][j][2 * r + 1]);
            *reinterpret_cast<uint32_t*>(obase + (long long)(c * kChunk + t) * inner + v) =
                pack_bf16x2(y0 * silu<__nv_bfloat16>(zz.x), y1 * silu<__nv_bfloat16>(zz.y));
          }
        }
      // ---- state after the chunk ----
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[j][e] *= keep;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        uint32_t xa[4], w1[4], w2[4], w3[4];          // x^T: rows v0 + g (0, 2), + 8 (1, 3); tokens 16 k + 2 tq (0, 1), + 8 (2, 3)
        ldsm4t(xa, sx + (k * 16 + (lane & 7) + (lane >> 4) * 8) * Sh::kXPitch + warp * 32 + ((lane >> 3) & 1) * 16);
#pragma unroll
        for (int q = 0; q < 2; ++q) {
          const int t = k * 16 + 2 * tq + 8 * q;
          const float x = sW[t], y = sW[t + 1];
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&xa[2 * q + r]));
            float f0 = f.x * x, f1 = f.y * y;
            w1[2 * q + r] = take_bf16(f0, f1);
            w2[2 * q + r] = take_bf16(f0, f1);
            w3[2 * q + r] = take_bf16(f0, f1);
          }
        }
#pragma unroll
        for (int j = 0; j < NT; j += 2) {
          uint32_t bb[4];                             // tokens 16 k.. of dimensions 8 j.. (0, 1), 8 j + 8.. (2, 3)
          ldsm4t(bb, sb + (k * 16 + (lane & 15)) * Sh::kCPitch + j * 16 + (lane >> 4) * 16);
          mma(s[j], w1, bb[0], bb[1]);
          mma(s[j + 1], w1, bb[2], bb[3]);
          mma(s[j], w2, bb[0], bb[1]);
          mma(s[j + 1], w2, bb[2], bb[3]);
          mma(s[j], w3, bb[0], bb[1]);
          mma(s[j + 1], w3, bb[2], bb[3]);
        }
      }
    }
    __syncthreads();
    if (STAGES == 1 && c + 1 < chunks) fetch(c + 1);
  }
  float* S = p.S + head * N * P;
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = 8 * j + 2 * tq + (e & 1), v = v0 + g + (e >> 1) * 8;
      if (d < N && v < P) S[(long long)d * P + v] = s[j][e];
    }
}

bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

bool chunks_ok(const Args& a) {
  return a.N % 8 == 0 && a.P % 8 == 0 && a.N <= 256 && a.ld % 8 == 0 && a.ld_x % 8 == 0 && al16(a.proj) && al16(a.xbc) &&
         al16(a.out) && al16(a.gates);
}

template <int NP, int STAGES>
int chunk_launch(const Args& a, cudaStream_t stream) {
  using Sh = ChunkShape<NP, STAGES>;
  static_assert(2 * (Sh::kSmem + 1024) <= 233472, "two CTAs per SM");
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(chunk_kernel<NP, STAGES>, cudaFuncAttributeMaxDynamicSharedMemorySize, Sh::kSmem) != cudaSuccess) {
      mfb_host::set_error("state_space: cannot raise the shared memory limit");
      return 10;
    }
    attr_set = true;
  }
  chunk_kernel<NP, STAGES><<<dim3((a.P + 63) / 64, a.H, a.B), 128, Sh::kSmem, stream>>>(a);
  return 0;
}

int in_chunks(const Args& a, int longest, cudaStream_t stream) {
  const dim3 grid((longest + kChunk - 1) / kChunk, a.B, (a.H + kGateHeads - 1) / kGateHeads);
  gates_kernel<__nv_bfloat16><<<grid, 32 * kGateHeads, 0, stream>>>(a);
  if (a.N <= 32) return chunk_launch<32, 2>(a, stream);
  if (a.N <= 64) return chunk_launch<64, 2>(a, stream);
  if (a.N <= 128) return chunk_launch<128, 2>(a, stream);
  return chunk_launch<256, 1>(a, stream);
}

template <typename T, int VEC>
void conv(Args a, cudaStream_t stream) {
  const int per = 128 * VEC;
  a.rows = 32;                                        // the rows in front of a run are read once more
  while (a.rows > 4 && (long long)((a.T + a.rows - 1) / a.rows) * ((a.channels() + per - 1) / per) < 148 * 4) a.rows /= 2;
  const dim3 grid((a.T + a.rows - 1) / a.rows, (a.channels() + per - 1) / per);
  if (a.taps <= 2) conv_kernel<T, VEC, 2><<<grid, 128, 0, stream>>>(a);
  else if (a.taps <= 4) conv_kernel<T, VEC, 4><<<grid, 128, 0, stream>>>(a);
  else if (VEC == 1) conv_kernel<T, 1, kMaxTaps><<<grid, 128, 0, stream>>>(a);
}

template <typename T>
void scan(const Args& a, cudaStream_t stream) {
  const dim3 grid((a.P + kCols - 1) / kCols, a.H, a.B);
  const int r = (a.N + kGroups - 1) / kGroups;
  if (r <= 8) scan_kernel<T, 8><<<grid, kScan, 0, stream>>>(a);
  else if (r <= 16) scan_kernel<T, 16><<<grid, kScan, 0, stream>>>(a);
  else if (r <= 32) scan_kernel<T, 32><<<grid, kScan, 0, stream>>>(a);
  else scan_kernel<T, 64><<<grid, kScan, 0, stream>>>(a);
}

template <typename T, int VEC>
int finish(const Args& a, cudaStream_t stream) {
  const int gw = a.inner() / a.norm_groups, nvec = gw / VEC;
  auto go = [&](auto kern, int k) {
    const int x = ((nvec + k - 1) / k + 31) / 32 * 32, y = x == 32 ? 4 : 1;
    const long long items = (long long)a.T * a.norm_groups;
    const long long ring = a.cu_q ? (long long)a.B * a.taps * ((a.channels() + kRingCols - 1) / kRingCols) : 0;
    kern<<<(unsigned)((items + y - 1) / y + ring), dim3(x, y), 0, stream>>>(a);
  };
  if (nvec <= 32) go(finish_kernel<T, VEC, 1>, 1);
  else if (nvec <= 64) go(finish_kernel<T, VEC, 2>, 2);
  else if (nvec <= 4096) go(finish_kernel<T, VEC, 4>, 4);
  else if (VEC == 1 && nvec <= 16384) go(finish_kernel<T, 1, 16>, 16);
  else { mfb_host::set_error("state_space: parts of %d columns", gw); return 1; }
  return 0;
}

template <typename T>
int run(Args a, int longest, cudaStream_t stream) {
  constexpr int V = 16 / sizeof(T);
  const int C = a.channels();
  if (a.cu_q) {
    const bool vec = a.inner() % V == 0 && C % V == 0 && a.ld % V == 0 && a.ld_x % V == 0 && al16(a.proj) && al16(a.xbc) &&
                     al16(a.ring) && al16(a.conv) && al16(a.conv_b) && C % 4 == 0 && a.taps <= 4;
    if (vec) conv<T, 4>(a, stream);
    else conv<T, 1>(a, stream);
    if (sizeof(T) == 2 && longest > 0 && chunks_ok(a)) {
      if (int rc = in_chunks(a, longest, stream)) return rc;
    } else scan<T>(a, stream);
  } else {
    const bool vec = a.P % 4 == 0;
    auto bytes = [&](int heads) { return (size_t)(2 * a.N + heads * (a.P + kDec * (vec ? 4 : 1))) * sizeof(float); };
    a.rows = 1;                                       // heads per CTA, as long as the GPU stays full
    while (a.rows < 4 && (a.H / a.G) % (a.rows * 2) == 0 && a.H / (a.rows * 2) * (long long)a.B >= 148 * 4 &&
           bytes(a.rows * 2) <= 32 * 1024) a.rows *= 2;
    const size_t smem = bytes(a.rows);
    if (smem > 48 * 1024) { mfb_host::set_error("state_space: N=%d P=%d", a.N, a.P); return 1; }
    const dim3 grid(a.H / a.rows, a.B);
    if (vec) decode_kernel<T, 4><<<grid, kDec, smem, stream>>>(a);
    else decode_kernel<T, 1><<<grid, kDec, smem, stream>>>(a);
  }
  const int gw = a.inner() / a.norm_groups;
  const bool vec = gw % V == 0 && gw % 4 == 0 && al16(a.out) && al16(a.norm);
  if (int rc = vec ? finish<T, V>(a, stream) : finish<T, 1>(a, stream)) return rc;
  return cudaGetLastError() == cudaSuccess ? 0 : 2;
}

}  // namespace ssm
}  // namespace mfb

extern "C" {
using namespace mfb;

// fp32 values of scratch for portions.
long long mfb_state_space_scratch_floats(int T, int H, int P, int N) { return (long long)T * H * 4 + 4; }

// See the head of this file. cu_q [B + 1] (device): portions, with scratch and xbc [T, H P + 2 G N] (rows ld_x apart); null: one row
// per slot (T == B). longest: rows of the longest portion. State sizes up to 512, head sizes up to 4096, up to 16 taps.
// f32 = 1: activations are fp32, else bf16.
int mfb_state_space(const void* proj, long long ld, const float* conv, const float* conv_b, const float* dt_bias, const float* a_log,
                    const float* d, const float* norm, void* ring, float* S, const int* cu_q, const int* context_lens,
                    const int* slots, float* scratch, void* xbc, void* out, long long ld_x, int T, int B, int H, int P, int N, int G,
                    int taps, int norm_groups, int longest, float eps, int f32, cudaStream_t stream) {
  if (T <= 0 || B <= 0) return 0;
  if (H < 1 || P < 1 || N < 1 || G < 1 || H % G || N > ssm::kMaxN || P > 4096 || H > 65535 || B > 65535 || taps < 1 ||
      taps > ssm::kMaxTaps || norm_groups < 1 || (H * P) % norm_groups || ld < 2LL * H * P + 2LL * G * N + H ||
      (!cu_q && T != B) || (cu_q && (!scratch || !xbc || ld_x < (long long)H * P + 2LL * G * N))) {
    mfb_host::set_error("state_space: T=%d B=%d H=%d P=%d N=%d G=%d taps=%d norm_groups=%d ld=%lld", T, B, H, P, N, G, taps,
                        norm_groups, ld);
    return 1;
  }
  ssm::Args a;
  a.proj = proj; a.ld = ld; a.conv = conv; a.conv_b = conv_b; a.dt_bias = dt_bias; a.a_log = a_log; a.d = d; a.norm = norm;
  a.ring = ring; a.S = S; a.cu_q = cu_q; a.context_lens = context_lens; a.slots = slots;
  a.gates = reinterpret_cast<float4*>(scratch); a.xbc = xbc; a.ld_x = ld_x; a.out = out;
  a.T = T; a.B = B; a.H = H; a.P = P; a.N = N; a.G = G; a.taps = taps; a.norm_groups = norm_groups; a.rows = 0; a.eps = eps;
  const int rc = f32 ? ssm::run<float>(a, longest, stream) : ssm::run<__nv_bfloat16>(a, longest, stream);
  if (rc == 2) mfb_host::set_error("state_space: launch failed");
  return rc;
}

}  // extern "C"
