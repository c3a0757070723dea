// Gated delta rule over ragged batches with a recurrent state per sequence slot (sm_100a). Per head, from token to token:
//
//   S <- g * S              S [D, DV] fp32; g: one decay per head, or one per head and key channel (rows of S)
//   u  = beta * (v - S^T k)
//   S <- S + k u^T
//   o  = S^T q
//
// q, k and v are projections that passed a short causal convolution over time and silu; q and k are unit vectors per head
// (q also times D^-1/2) and G of them serve H heads. o is normalised over DV, weighted, and gated (silu or sigmoid).
// Everything from the convolution's result to o is fp32.
//
// State of slot b: S [H, D, DV] and the last `taps` inputs of the convolution, a ring in which position p has place
// p % taps. Slot b belongs to row b of the batch. Nothing has to be cleared when a slot changes hands: a portion that starts
// at position 0 reads neither S nor the ring, and no position below 0 is ever read.
//
// A batch is ragged: sequence b brings the rows cu_q[b] .. cu_q[b + 1] - 1, which end at position context_lens[b] - 1.
// Portions run as prepare (convolutions, unit vectors) and decays -> scan (the recurrence) -> gate_out. A decode step (one row
// per slot) is one kernel, delta_decode.
//
// The scan walks the tokens in fp32 on the FMA pipes, since the state and all that enters it are 32-bit by design. Columns of
// S are independent: a CTA takes a range of the columns of one head of one sequence, L lanes share a column, and a thread
// keeps R rows of C columns in registers for the whole portion, as pairs for the packed fp32 instructions.
#include <type_traits>

#include "common.cuh"

namespace mfb {
namespace dlt {

__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
template <int VEC> __device__ __forceinline__ void ldv(const float* p, float (&v)[VEC]) {
  if constexpr (VEC == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  } else {
    v[0] = *p;
  }
}
template <int VEC> __device__ __forceinline__ void ldv(const __nv_bfloat16* p, float (&v)[VEC]) {
  if constexpr (VEC == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
  } else {
    v[0] = ld(p);
  }
}
template <int VEC> __device__ __forceinline__ void stv(float* p, const float (&v)[VEC]) {
  if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *p = v[0];
}
template <int VEC> __device__ __forceinline__ void stv(__nv_bfloat16* p, const float (&v)[VEC]) {
  if constexpr (VEC == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
  else st(p, v[0]);
}

// (an overflowing exponential gives a quotient of zero)
__device__ __forceinline__ float sigmoidf(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float siluf(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float softplusf(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float decayf(float a_log, float x) { return expf(-expf(a_log) * softplusf(x)); }

struct Args {
  const void* x;            // [T, >= 2 G D + H DV] (pitch ld): inputs of the convolution, q | k | v
  long long ld;
  const void* b;            // [T, H] (pitch ld): raw beta
  const void* a;            // raw decay: [T, H] or [T, H D] (pitch ld_a)
  long long ld_a;
  const void* gate;         // [T, H DV] (pitch ld_gate)
  long long ld_gate;
  const float* conv;        // [taps, 2 G D + H DV], the last row belongs to the current token
  const float* a_log;       // [H]
  const float* dt_bias;     // [H] or [H D]
  const float* norm;        // [DV]
  void* ring;               // [slots, taps, 2 G D + H DV] type T
  float* state;             // [slots, H, D, DV]
  const int* cu_q;          // [B + 1] (portions)
  const int* context_lens;  // [B]
  const int* slots;         // [B] cache slot of the row, negative: idle (decode)
  float* qk;                // scratch [T, G, 2, D]: unit q (scaled), unit k
  float* v;                 // scratch [T, H, DV]
  float* beta;              // scratch [T, H]
  float* g;                 // scratch [T, H] or [T, H, D]
  float* o;                 // scratch [T, H, DV]
  void* out;                // [T, H DV] type T (pitch ld_out)
  long long ld_out;
  int T, B, H, G, D, DV, taps, by_channel, gate_silu;
  float eps, out_scale;
};

// sequence of row r (the last one that starts at or before it and is not empty there)
__device__ __forceinline__ int sequence_of(const int* cu_q, int B, int r) {
  int lo = 0, hi = B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) / 2;
    if (cu_q[mid] <= r) lo = mid; else hi = mid - 1;
  }
  return lo;
}

constexpr int kRun = 8;                // consecutive rows of a warp in `prepare`

// silu(convolution) of channels c .. c + VEC - 1 at row r; `local` rows of the portion lie before r, `pos` is its position
template <typename T, int VEC>
__device__ __forceinline__ void conv_silu(const Args& p, const T* ring, long long r, int local, int pos, int c, int C, float (&acc)[VEC]) {
#pragma unroll
  for (int i = 0; i < VEC; ++i) acc[i] = 0.f;
  for (int d = p.taps - 1; d >= 0; --d) {
    if (d > pos) continue;
    float xv[VEC], wv[VEC];
    if (d <= local) ldv<VEC>(reinterpret_cast<const T*>(p.x) + (r - d) * p.ld + c, xv);
    else ldv<VEC>(ring + (long long)((pos - d) % p.taps) * C + c, xv);
    ldv<VEC>(p.conv + (long long)(p.taps - 1 - d) * C + c, wv);
#pragma unroll
    for (int i = 0; i < VEC; ++i) acc[i] = fmaf(xv[i], wv[i], acc[i]);
  }
#pragma unroll
  for (int i = 0; i < VEC; ++i) acc[i] = siluf(acc[i]);
}

// The same for four neighbouring channels of a run of rows and at most four taps, in registers: the run's inputs are fetched
// ahead, a window holds the three before the current one, and the weights stay.
template <typename T>
struct ConvRun {
  typedef typename std::conditional<sizeof(T) == 2, uint2, float4>::type Raw;
  Raw x[kRun];
  float w[4][4], before[3][4];          // w[d]: weight of the input d rows back
  __device__ __forceinline__ static void unpack(const Raw& r, float (&v)[4]) { ldv<4>(reinterpret_cast<const T*>(&r), v); }
  __device__ __forceinline__ void open(const Args& p, int r0, int c, int C) {
#pragma unroll
    for (int i = 0; i < kRun; ++i)
      if (r0 + i < p.T) x[i] = *reinterpret_cast<const Raw*>(reinterpret_cast<const T*>(p.x) + (long long)(r0 + i) * p.ld + c);
#pragma unroll
    for (int d = 0; d < 4; ++d) {
      if (d < p.taps) ldv<4>(p.conv + (long long)(p.taps - 1 - d) * C + c, w[d]);
      else { w[d][0] = w[d][1] = w[d][2] = w[d][3] = 0.f; }
    }
  }
  // the inputs before row r (first of the run or of its sequence)
  __device__ __forceinline__ void rewind(const Args& p, const T* ring, long long r, int local, int pos, int c, int C) {
#pragma unroll
    for (int d = 1; d < 4; ++d) {
      if (d < p.taps && d <= pos) {
        if (d <= local) ldv<4>(reinterpret_cast<const T*>(p.x) + (r - d) * p.ld + c, before[d - 1]);
        else ldv<4>(ring + (long long)((pos - d) % p.taps) * C + c, before[d - 1]);
      } else {
        before[d - 1][0] = before[d - 1][1] = before[d - 1][2] = before[d - 1][3] = 0.f;
      }
    }
  }
  __device__ __forceinline__ void next(const Raw& raw, float (&out)[4]) {
    float cur[4];
    unpack(raw, cur);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      float a = fmaf(before[2][i], w[3][i], before[1][i] * w[2][i]);
      a = fmaf(cur[i], w[0][i], fmaf(before[0][i], w[1][i], a));
      before[2][i] = before[1][i]; before[1][i] = before[0][i]; before[0][i] = cur[i];
      out[i] = siluf(a);
    }
  }
};

// One warp per unit and run of rows; units: G heads of q and G of k (made unit vectors, q also scaled), H heads of v. FAST: VEC
// 4, heads up to 128, at most four taps.
template <typename T, int VEC, int NJ, bool FAST>
__global__ void __launch_bounds__(128) prepare_kernel(const Args p) {
  const int unit = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (unit >= 2 * p.G + p.H) return;
  const int r0 = blockIdx.x * kRun, r1 = min(r0 + kRun, p.T);
  const int C = 2 * p.G * p.D + p.H * p.DV;
  const bool is_q = unit < p.G, is_v = unit >= 2 * p.G;
  const int size = is_v ? p.DV : p.D, c0 = is_v ? 2 * p.G * p.D + (unit - 2 * p.G) * p.DV : unit * p.D;
  float* dst;
  long long pitch;
  if (is_v) {
    pitch = (long long)p.H * p.DV;
    dst = p.v + (unit - 2 * p.G) * p.DV;
  } else {
    pitch = (long long)p.G * 2 * p.D;
    dst = p.qk + (is_q ? unit * 2 : (unit - p.G) * 2 + 1) * p.D;
  }
  const float scale = is_q ? 1.f / sqrtf((float)p.D) : 1.f;
  int b = sequence_of(p.cu_q, p.B, r0);
  ConvRun<T> run;
  const bool on = lane * 4 < size;
  if constexpr (FAST) {
    if (on) run.open(p, r0, c0 + lane * 4, C);
  }
#pragma unroll
  for (int ri = 0; ri < kRun; ++ri) {
    const int r = r0 + ri;
    if (r >= r1) break;
    while (r >= p.cu_q[b + 1]) ++b;
    const int local = r - p.cu_q[b], pos = p.context_lens[b] - (p.cu_q[b + 1] - r);
    const T* ring = reinterpret_cast<const T*>(p.ring) + (long long)b * p.taps * C;
    if constexpr (FAST) {
      if (on && (ri == 0 || local == 0)) run.rewind(p, ring, r, local, pos, c0 + lane * 4, C);
    }
    float v[NJ][VEC];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int d = (lane + 32 * j) * VEC;
      if (d < size) {
        if constexpr (FAST) run.next(run.x[ri], v[j]);
        else conv_silu<T, VEC>(p, ring, r, local, pos, c0 + d, C, v[j]);
#pragma unroll
        for (int i = 0; i < VEC; ++i) ss = fmaf(v[j][i], v[j][i], ss);
      }
    }
    float f = 1.f;
    if (!is_v) f = scale / sqrtf(warp_sum(ss) + 1e-6f);
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int d = (lane + 32 * j) * VEC;
      if (d < size) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[j][i] *= f;
        stv<VEC>(dst + r * pitch + d, v[j]);
      }
    }
  }
}

// beta [T, H] and the decays [T, H] or [T, H, D], VEC channels per thread
template <typename T, int VEC>
__global__ void __launch_bounds__(256) decay_kernel(const Args p) {
  const int per = p.by_channel ? p.D / VEC : 1;
  const long long n = (long long)p.T * p.H * per;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const long long rh = i / per, r = rh / p.H;
    const int h = (int)(rh - r * p.H), d = (int)(i - rh * per) * VEC;
    if (d == 0) p.beta[rh] = sigmoidf(ld(reinterpret_cast<const T*>(p.b) + r * p.ld + h));
    const T* a = reinterpret_cast<const T*>(p.a) + r * p.ld_a;
    if (p.by_channel) {
      float v[VEC], t[VEC];
      ldv<VEC>(a + h * p.D + d, v);
      ldv<VEC>(p.dt_bias + h * p.D + d, t);
      const float al = p.a_log[h];
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] = decayf(al, v[e] + t[e]);
      stv<VEC>(p.g + rh * p.D + d, v);
    } else {
      p.g[rh] = decayf(p.a_log[h], ld(a + h) + p.dt_bias[h]);
    }
  }
}

// ---- the recurrence -----------------------------------------------------------------------------------------------------
__device__ __forceinline__ uint64_t pack2(float lo, float hi) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ void unpack2(uint64_t v, float& lo, float& hi) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
constexpr int kComputeThreads = 128;
constexpr int kFeedWarps = 2;          // warps that load and prepare the vectors of the pairs ahead
constexpr int kScanThreads = kComputeThreads + 32 * kFeedWarps;
constexpr int kPairs = 4;              // pairs of tokens per stage (two stages)
constexpr int kTile = 2 * kPairs;

// vectors of a pair of tokens in a stage: with decays per channel k1 g1, q1 g1, k2 g1 g2, q2 g1 g2, k1 g2, k2, g1 g2; with one
// decay k1, q1, k2, q2
template <int R, int L, int C, bool CH>
struct ScanShape {
  static constexpr int DP = R * L;                          // padded key size
  static constexpr int kGroups = kComputeThreads / L;
  static constexpr int kCols = kGroups * C;                 // columns of a CTA
  static constexpr int kVecs = CH ? 7 : 4;
  static constexpr int kStage = kPairs * (kVecs * DP + 2 * kCols + 8);      // floats; 8: beta1, q1 k1, beta2, q2 k2, c, q2 k1, g1, g2
};

// sum over the L lanes of a column group of N values per lane; lane l is left with values l, l + L, ... (N / L of them), or,
// where N < L, with value l N / L: halves are exchanged as long as a lane holds more than one
template <int N, int L>
__device__ __forceinline__ void reduce_scatter(float (&v)[N], int ln) {
  int n = N;
#pragma unroll
  for (int d = L / 2; d > 0; d >>= 1) {
    if (n > 1) {
      n /= 2;
      const bool up = ln & d;
#pragma unroll
      for (int i = 0; i < N / 2; ++i) {
        if (i < n) {
          const float keep = up ? v[i + n] : v[i], give = up ? v[i] : v[i + n];
          v[i] = keep + __shfl_xor_sync(0xffffffffu, give, d);
        }
      }
    } else {
      v[0] += __shfl_xor_sync(0xffffffffu, v[0], d);
    }
  }
}

// Two tokens at a time. With S the state before them, A1 = S^T (g1 k1), A2 = S^T (g1 g2 k2) and B1, B2 the same of q:
//   u1 = beta1 (v1 - A1)                 o1 = B1 + (q1 . k1) u1
//   u2 = beta2 (v2 - A2 - c u1)          o2 = B2 + (q2 . g2 k1) u1 + (q2 . k2) u2        c = k2 . g2 k1
//   S <- g1 g2 S + (g2 k1) u1^T + k2 u2^T
// which is the same recurrence with seven instead of eight operations per element and pair, and one instead of two points at
// which the lanes of a column wait for one another. R rows of C columns per thread, L lanes per column; CH: decays per key
// channel. vec: D, DV and the scratch rows allow 16-byte accesses. While the compute warps work on one stage of pairs, the
// feed warps fetch and prepare the next.
template <typename T, int R, int L, int C, bool CH>
__global__ void __launch_bounds__(kScanThreads, 2) scan_kernel(const Args p, int vec) {
  using S = ScanShape<R, L, C, CH>;
  constexpr int DP = S::DP, COLS = S::kCols, GROUPS = S::kGroups, VECS = S::kVecs;
  const int b = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * COLS;
  const int r0 = p.cu_q[b], n = p.cu_q[b + 1] - r0;
  if (n <= 0) return;
  const int end = p.context_lens[b], start = end - n;
  const int D = p.D, DV = p.DV, H = p.H, kvh = h / (H / p.G);
  if (blockIdx.x == 0 && h == 0) {
    // the convolution's inputs of the last positions (`prepare`, which read the old ones, has finished)
    const int ch = 2 * p.G * D + H * DV, keep = min(n, p.taps);
    T* ring = reinterpret_cast<T*>(p.ring) + (long long)b * p.taps * ch;
    for (int i = 0; i < keep; ++i) {
      const int pos = end - keep + i;
      const T* src = reinterpret_cast<const T*>(p.x) + (long long)(r0 + n - keep + i) * p.ld;
      for (int c = threadIdx.x; c < ch; c += kScanThreads) ring[(long long)(pos % p.taps) * ch + c] = src[c];
    }
  }
  extern __shared__ __align__(16) float sh[];        // [2][kStage]: vectors of the pairs, v, scalars
  const int lane = threadIdx.x & 31;
  const int tiles = (n + kTile - 1) / kTile;

  if (threadIdx.x >= kComputeThreads) {
    // ------------------------------ feed ------------------------------
    constexpr int NJ = (DP + 127) / 128, PW = kPairs / kFeedWarps, VN = (2 * COLS + 127) / 128;
    const int fw = (threadIdx.x - kComputeThreads) >> 5;
    float k[PW][2][NJ][4], q[PW][2][NJ][4], g[PW][2][CH ? NJ : 1][4], v[PW][VN][4];
    float bs[PW], gs[PW];                            // lanes 0 and 1: beta and decay (without CH) of the two tokens
    auto four = [&](const float* src, int at, int size, float fill, float (&o)[4]) {
      if (at + 3 < size && vec) { ldv<4>(src + at, o); return; }
#pragma unroll
      for (int e = 0; e < 4; ++e) o[e] = at + e < size ? src[at + e] : fill;
    };
    auto fetch = [&](int tile) {
#pragma unroll
      for (int w = 0; w < PW; ++w) {
        const int t0 = tile * kTile + 2 * (fw + w * kFeedWarps);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const bool there = t0 + e < n;             // an odd last token is paired with one that changes nothing
          const long long row = r0 + (there ? t0 + e : n - 1);
          const float* src = p.qk + (row * p.G + kvh) * 2 * D;
#pragma unroll
          for (int j = 0; j < NJ; ++j) {
            const int d = (lane + 32 * j) * 4;
            four(src, d, there ? D : 0, 0.f, q[w][e][j]);
            four(src + D, d, there ? D : 0, 0.f, k[w][e][j]);
            if constexpr (CH) four(p.g + (row * H + h) * D, d, there ? D : 0, 1.f, g[w][e][j]);
          }
        }
#pragma unroll
        for (int i = 0; i < VN; ++i) {
          const int at = (lane + 32 * i) * 4, e = at / COLS, c = at % COLS;
          if (e < 2) four(p.v + ((long long)(r0 + min(t0 + e, n - 1)) * H + h) * DV, col0 + c, DV, 0.f, v[w][i]);
        }
        if (lane < 2) {
          const bool there = t0 + lane < n;
          const long long at = (long long)(r0 + (there ? t0 + lane : n - 1)) * H + h;
          bs[w] = there ? p.beta[at] : 0.f;
          gs[w] = !CH && there ? p.g[at] : 1.f;
        }
      }
    };
    auto put = [&](int tile) {
      float* stage = sh + (tile & 1) * S::kStage;
#pragma unroll
      for (int w = 0; w < PW; ++w) {
        const int j2 = fw + w * kFeedWarps;
        float* vecs = stage + j2 * VECS * DP;
        float kk = 0.f, qk = 0.f, own1 = 0.f, own2 = 0.f;
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
          const int d = (lane + 32 * j) * 4;
          if (d < DP) {
            float o[7][4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const float k1 = k[w][0][j][e], q1 = q[w][0][j][e], k2 = k[w][1][j][e], q2 = q[w][1][j][e];
              float w1 = k1;
              if constexpr (CH) {
                const float g1 = g[w][0][j][e], g2 = g[w][1][j][e], gg = g1 * g2;
                w1 = k1 * g2;
                o[0][e] = k1 * g1; o[1][e] = q1 * g1; o[2][e] = k2 * gg; o[3][e] = q2 * gg;
                o[4][e] = w1; o[5][e] = k2; o[6][e] = gg;
              } else {
                o[0][e] = k1; o[1][e] = q1; o[2][e] = k2; o[3][e] = q2;
              }
              kk = fmaf(k2, w1, kk);
              qk = fmaf(q2, w1, qk);
              own1 = fmaf(q1, k1, own1);
              own2 = fmaf(q2, k2, own2);
            }
#pragma unroll
            for (int x = 0; x < VECS; ++x) stv<4>(vecs + x * DP + d, o[x]);
          }
        }
        kk = warp_sum(kk);
        qk = warp_sum(qk);
        own1 = warp_sum(own1);
        own2 = warp_sum(own2);
        float* vs = stage + kPairs * VECS * DP + j2 * 2 * COLS;
#pragma unroll
        for (int i = 0; i < VN; ++i) {
          const int at = (lane + 32 * i) * 4;
          if (at < 2 * COLS) stv<4>(vs + at, v[w][i]);
        }
        float* ss = stage + kPairs * (VECS * DP + 2 * COLS) + j2 * 8;
        const float g2 = __shfl_sync(0xffffffffu, gs[w], 1);
        if (lane < 2) { ss[2 * lane] = bs[w]; ss[2 * lane + 1] = lane ? own2 : own1; ss[6 + lane] = gs[w]; }
        if (lane == 0) { ss[4] = CH ? kk : kk * g2; ss[5] = CH ? qk : qk * g2; }
      }
    };
    fetch(0);
    put(0);
    if (tiles > 1) fetch(1);
    __syncthreads();
    for (int tile = 0; tile < tiles; ++tile) {
      if (tile + 1 < tiles) put(tile + 1);
      if (tile + 2 < tiles) fetch(tile + 2);
      __syncthreads();
    }
    return;
  }

  // ------------------------------ compute ------------------------------
  const int ln = threadIdx.x % L, grp = threadIdx.x / L;
  // rows of a thread: (i * L + ln) * 4 .. + 3 for i < R / 4, as pairs
  uint64_t s[C][R / 2];
  float* state = p.state + ((long long)b * H + h) * D * DV;
#pragma unroll
  for (int c = 0; c < C; ++c) {
    const int col = col0 + grp + GROUPS * c;
#pragma unroll
    for (int i = 0; i < R / 2; ++i) {
      float v[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int row = ((i >> 1) * L + ln) * 4 + (i & 1) * 2 + e;
        v[e] = (start > 0 && row < D && col < DV) ? state[(long long)row * DV + col] : 0.f;
      }
      s[c][i] = pack2(v[0], v[1]);
    }
  }
  // after the exchange of partial sums a lane computes one column (C <= L), or C / L of them
  constexpr int OWN = C > L ? C / L : 1;
  __syncthreads();
  for (int tile = 0; tile < tiles; ++tile) {
    const float* stage = sh + (tile & 1) * S::kStage;
    const int m = min(kTile, n - tile * kTile);
    float* orow = p.o + ((long long)(r0 + tile * kTile) * H + h) * DV;
    for (int j = 0; 2 * j < m; ++j) {
      const float* vec1 = stage + j * VECS * DP + ln * 4;
      uint64_t acc[C][4];
#pragma unroll
      for (int c = 0; c < C; ++c)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[c][e] = 0;
#pragma unroll
      for (int i = 0; i < R / 4; ++i) {
        const ulonglong2 k1 = *reinterpret_cast<const ulonglong2*>(vec1 + i * L * 4);
        const ulonglong2 q1 = *reinterpret_cast<const ulonglong2*>(vec1 + DP + i * L * 4);
        const ulonglong2 k2 = *reinterpret_cast<const ulonglong2*>(vec1 + 2 * DP + i * L * 4);
        const ulonglong2 q2 = *reinterpret_cast<const ulonglong2*>(vec1 + 3 * DP + i * L * 4);
#pragma unroll
        for (int c = 0; c < C; ++c) {
          acc[c][0] = fma2(s[c][2 * i], k1.x, acc[c][0]);
          acc[c][1] = fma2(s[c][2 * i], q1.x, acc[c][1]);
          acc[c][2] = fma2(s[c][2 * i], k2.x, acc[c][2]);
          acc[c][3] = fma2(s[c][2 * i], q2.x, acc[c][3]);
        }
#pragma unroll
        for (int c = 0; c < C; ++c) {
          acc[c][0] = fma2(s[c][2 * i + 1], k1.y, acc[c][0]);
          acc[c][1] = fma2(s[c][2 * i + 1], q1.y, acc[c][1]);
          acc[c][2] = fma2(s[c][2 * i + 1], k2.y, acc[c][2]);
          acc[c][3] = fma2(s[c][2 * i + 1], q2.y, acc[c][3]);
        }
      }
      const float* ss = stage + kPairs * (VECS * DP + 2 * COLS) + j * 8;
      const float4 bb = *reinterpret_cast<const float4*>(ss), cg = *reinterpret_cast<const float4*>(ss + 4);
      const float g1 = CH ? 1.f : cg.z, g12 = CH ? 1.f : cg.z * cg.w;
      float sums[4][C];
#pragma unroll
      for (int c = 0; c < C; ++c)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          float x, y;
          unpack2(acc[c][e], x, y);
          sums[e][c] = x + y;
        }
#pragma unroll
      for (int e = 0; e < 4; ++e) reduce_scatter<C, L>(sums[e], ln);
      // this lane's column(s)
      float u1[OWN], u2[OWN];
#pragma unroll
      for (int o = 0; o < OWN; ++o) {
        const int c = C > L ? ln * OWN + o : (ln * C) / L;
        const int lc = grp + GROUPS * c, col = col0 + lc;
        const float* vp = stage + kPairs * VECS * DP + j * 2 * COLS + lc;
        u1[o] = bb.x * (vp[0] - g1 * sums[0][o]);
        u2[o] = bb.z * (vp[COLS] - g12 * sums[2][o] - cg.x * u1[o]);
        if (col < DV && (C >= L || ln % (L / C) == 0)) {
          orow[(long long)(2 * j) * H * DV + col] = fmaf(u1[o], bb.y, g1 * sums[1][o]);
          if (2 * j + 1 < m) orow[(long long)(2 * j + 1) * H * DV + col] = fmaf(u2[o], bb.w, fmaf(cg.y, u1[o], g12 * sums[3][o]));
        }
        if (!CH) u1[o] *= cg.w;
      }
      const uint64_t g2 = pack2(g12, g12);
      const float* w1p = CH ? vec1 + 4 * DP : vec1;
      const float* w2p = CH ? vec1 + 5 * DP : vec1 + 2 * DP;
      const float* gp = vec1 + 6 * DP;
      uint64_t x1[C], x2[C];
#pragma unroll
      for (int c = 0; c < C; ++c) {
        const int src = (lane & ~(L - 1)) + (C > L ? c / OWN : c * (L / C));
        const float y1 = __shfl_sync(0xffffffffu, u1[C > L ? c % OWN : 0], src), y2 = __shfl_sync(0xffffffffu, u2[C > L ? c % OWN : 0], src);
        x1[c] = pack2(y1, y1);
        x2[c] = pack2(y2, y2);
      }
#pragma unroll
      for (int i = 0; i < R / 4; ++i) {
        const ulonglong2 w1 = *reinterpret_cast<const ulonglong2*>(w1p + i * L * 4);
        const ulonglong2 w2 = *reinterpret_cast<const ulonglong2*>(w2p + i * L * 4);
        ulonglong2 g4;
        if (CH) g4 = *reinterpret_cast<const ulonglong2*>(gp + i * L * 4);
#pragma unroll
        for (int c = 0; c < C; ++c) {
          s[c][2 * i] = fma2(w2.x, x2[c], fma2(w1.x, x1[c], mul2(s[c][2 * i], CH ? g4.x : g2)));
          s[c][2 * i + 1] = fma2(w2.y, x2[c], fma2(w1.y, x1[c], mul2(s[c][2 * i + 1], CH ? g4.y : g2)));
        }
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int c = 0; c < C; ++c) {
    const int col = col0 + grp + GROUPS * c;
#pragma unroll
    for (int i = 0; i < R / 2; ++i) {
      float v[2];
      unpack2(s[c][i], v[0], v[1]);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int row = ((i >> 1) * L + ln) * 4 + (i & 1) * 2 + e;
        if (row < D && col < DV) state[(long long)row * DV + col] = v[e];
      }
    }
  }
}

// ---- norm and gate of the read-out: a warp per row and head -----------------------------------------------------------------
template <typename T, int VEC, int NJ>
__global__ void __launch_bounds__(128) gate_out_kernel(const Args p) {
  const long long item = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (item >= (long long)p.T * p.H) return;
  const int lane = threadIdx.x & 31;
  const long long r = item / p.H;
  const int h = (int)(item - r * p.H);
  const float* o = p.o + item * p.DV;
  const T* gate = reinterpret_cast<const T*>(p.gate) + r * p.ld_gate + h * p.DV;
  T* out = reinterpret_cast<T*>(p.out) + r * p.ld_out + h * p.DV;
  float v[NJ][VEC];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    const int d = (lane + 32 * j) * VEC;
    if (d < p.DV) {
      ldv<VEC>(o + d, v[j]);
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss = fmaf(v[j][i], v[j][i], ss);
    }
  }
  const float rstd = 1.f / sqrtf(warp_sum(ss) / p.DV + p.eps) * p.out_scale;
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    const int d = (lane + 32 * j) * VEC;
    if (d < p.DV) {
      float w[VEC], z[VEC];
      ldv<VEC>(p.norm + d, w);
      ldv<VEC>(gate + d, z);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[j][i] = v[j][i] * rstd * w[i] * (p.gate_silu ? siluf(z[i]) : sigmoidf(z[i]));
      stv<VEC>(out + d, v[j]);
    }
  }
}

// ---- decode: one row per slot, one CTA per head ---------------------------------------------------------------------------------
// Threads form TY row groups of TX lanes; a lane holds four neighbouring columns of NR rows. D * DV <= 4 NT NR. FAST (at most
// four taps, 2 D + DV <= NI NT, D and DV <= NT): every input is on its way before the first one is used, the state last, so that
// a CTA waits for memory once.
template <typename T, int NT, int NR, int NI, bool FAST>
__global__ void __launch_bounds__(NT, NR > 8 && NT > 256 ? 1 : 2) delta_decode_kernel(const Args p, int tx_log2) {
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int slot = p.slots[b], pos = p.context_lens[b] - 1;
  const int D = p.D, DV = p.DV, H = p.H, reps = H / p.G, kvh = h / reps;
  T* out = reinterpret_cast<T*>(p.out) + (long long)b * p.ld_out + h * DV;
  if (slot < 0) {                              // idle slot: the state stays, the row is defined
    for (int i = tid; i < DV; i += NT) st(out + i, 0.f);
    return;
  }
  const int TX = 1 << tx_log2, TY = NT >> tx_log2, tx = tid & (TX - 1), ty = tid >> tx_log2;
  const int warp = tid >> 5, lane = tid & 31;
  const int C = 2 * p.G * D + H * DV, items = 2 * D + DV;
  T* ring = reinterpret_cast<T*>(p.ring) + (long long)b * p.taps * C;
  const T* x = reinterpret_cast<const T*>(p.x) + (long long)b * p.ld;
  const T* a = reinterpret_cast<const T*>(p.a) + (long long)b * p.ld_a;
  const T* gate = reinterpret_cast<const T*>(p.gate) + (long long)b * p.ld_gate + h * DV;
  auto channel = [&](int i) {
    return i < D ? kvh * D + i : (i < 2 * D ? (p.G + kvh) * D + i - D : 2 * p.G * D + h * DV + i - 2 * D);
  };
  T xr[NI][4], ar, zr, br = reinterpret_cast<const T*>(p.b)[(long long)b * p.ld + h];
  st(&ar, 0.f); st(&zr, 0.f);
  float wr[NI][4], dt = 0.f, nw = 0.f;
  const float al = p.a_log[h];
  if constexpr (FAST) {
#pragma unroll
    for (int j = 0; j < NI; ++j) {
      const int i = tid + NT * j, c = i < items ? channel(i) : 0;
#pragma unroll
      for (int d = 0; d < 4; ++d) {
        st(&xr[j][d], 0.f);
        wr[j][d] = 0.f;
        if (i < items && d < p.taps && d <= pos) {
          xr[j][d] = d == 0 ? x[c] : ring[(long long)((pos - d) % p.taps) * C + c];
          wr[j][d] = p.conv[(long long)(p.taps - 1 - d) * C + c];
        }
      }
    }
    if (tid < D) {
      ar = a[p.by_channel ? h * D + tid : h];
      dt = p.dt_bias[p.by_channel ? h * D + tid : h];
    }
    if (tid < DV) { zr = gate[tid]; nw = p.norm[tid]; }
  }
  float* state = p.state + ((long long)b * H + h) * D * DV;
  const int col = tx * 4;
  float4 s[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int row = ty + TY * i;
    s[i] = (pos > 0 && row < D && col < DV) ? *reinterpret_cast<const float4*>(state + (long long)row * DV + col)
                                            : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  extern __shared__ __align__(16) float sh[];
  float* s_u = sh;                             // [DV] (16-byte aligned: DV is a multiple of 4)
  float* s_q = s_u + DV;                       // [D]
  float* s_k = s_q + D;                        // [D]
  float* s_v = s_k + D;                        // [DV], later o
  float* s_g = s_v + DV;                       // [D]
  float* s_red = s_g + D;                      // [NT / 32] + 2 x [TY][4 TX]
  // the ring has a place for the current input that no token up to this one reads: heads that share q and k do not race
  if constexpr (FAST) {
#pragma unroll
    for (int j = 0; j < NI; ++j) {
      const int i = tid + NT * j;
      if (i < items) {
        float acc = 0.f;
#pragma unroll
        for (int d = 3; d >= 0; --d) acc = fmaf(ld(&xr[j][d]), wr[j][d], acc);
        s_q[i] = siluf(acc);
        if (i >= 2 * D || h % reps == 0) ring[(long long)(pos % p.taps) * C + channel(i)] = xr[j][0];
      }
    }
    if (tid < D) s_g[tid] = decayf(al, ld(&ar) + dt);
  } else {
    for (int i = tid; i < items; i += NT) {
      const int c = channel(i);
      float v[1];
      conv_silu<T, 1>(p, ring, b, 0, pos, c, C, v);
      s_q[i] = v[0];
      if (i >= 2 * D || h % reps == 0) ring[(long long)(pos % p.taps) * C + c] = x[c];
    }
    for (int i = tid; i < D; i += NT) {
      const int c = p.by_channel ? h * D + i : h;
      s_g[i] = decayf(al, ld(a + c) + p.dt_bias[c]);
    }
  }
  const float beta = sigmoidf(ld(&br));
  __syncthreads();
  float qq = 0.f, kk = 0.f, qk = 0.f;
  for (int i = lane; i < D; i += 32) {
    qq = fmaf(s_q[i], s_q[i], qq);
    kk = fmaf(s_k[i], s_k[i], kk);
    qk = fmaf(s_q[i], s_k[i], qk);
  }
  qq = warp_sum(qq); kk = warp_sum(kk); qk = warp_sum(qk);
  const float rq = 1.f / sqrtf(qq + 1e-6f) / sqrtf((float)D), rk = 1.f / sqrtf(kk + 1e-6f);
  float av[4] = {0.f, 0.f, 0.f, 0.f}, bv[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int row = ty + TY * i;
    if (row < D) {
      const float g = s_g[row], k = s_k[row] * rk, q = s_q[row] * rq;
      s[i].x *= g; s[i].y *= g; s[i].z *= g; s[i].w *= g;
      av[0] = fmaf(s[i].x, k, av[0]); av[1] = fmaf(s[i].y, k, av[1]); av[2] = fmaf(s[i].z, k, av[2]); av[3] = fmaf(s[i].w, k, av[3]);
      bv[0] = fmaf(s[i].x, q, bv[0]); bv[1] = fmaf(s[i].y, q, bv[1]); bv[2] = fmaf(s[i].z, q, bv[2]); bv[3] = fmaf(s[i].w, q, bv[3]);
    }
  }
  float* red_a = s_red + NT / 32;
  float* red_b = red_a + NT * 4;
#pragma unroll
  for (int i = 0; i < 4; ++i) { red_a[ty * TX * 4 + col + i] = av[i]; red_b[ty * TX * 4 + col + i] = bv[i]; }
  __syncthreads();
  float ss = 0.f;
  for (int c = tid; c < DV; c += NT) {
    float sa = 0.f, sb = 0.f;
    for (int y = 0; y < TY; ++y) { sa += red_a[y * TX * 4 + c]; sb += red_b[y * TX * 4 + c]; }
    const float u = beta * (s_v[c] - sa);
    const float o = fmaf(u, qk * rq * rk, sb);
    s_u[c] = u;
    s_v[c] = o;
    ss = fmaf(o, o, ss);
  }
  ss = warp_sum(ss);
  if (lane == 0) s_red[warp] = ss;
  __syncthreads();
  if (col < DV) {
    const float4 u = *reinterpret_cast<const float4*>(s_u + col);
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int row = ty + TY * i;
      if (row < D) {
        const float k = s_k[row] * rk;
        *reinterpret_cast<float4*>(state + (long long)row * DV + col) =
            make_float4(fmaf(k, u.x, s[i].x), fmaf(k, u.y, s[i].y), fmaf(k, u.z, s[i].z), fmaf(k, u.w, s[i].w));
      }
    }
  }
  float tot = 0.f;
#pragma unroll
  for (int i = 0; i < NT / 32; ++i) tot += s_red[i];
  const float rstd = 1.f / sqrtf(tot / DV + p.eps) * p.out_scale;
  for (int c = tid; c < DV; c += NT) {
    const float z = FAST ? ld(&zr) : ld(gate + c), w = FAST ? nw : p.norm[c];
    st(out + c, s_v[c] * rstd * w * (p.gate_silu ? siluf(z) : sigmoidf(z)));
  }
}

// ---- launchers --------------------------------------------------------------------------------------------------------------------
bool al(const void* p, int bytes) { return (reinterpret_cast<uintptr_t>(p) & (bytes - 1)) == 0; }

int fail(const char* what) {
  if (cudaGetLastError() != cudaSuccess) { mfb_host::set_error("delta_rule: launch of %s failed", what); return 2; }
  return 0;
}

template <typename T>
int prepare(const Args& p, cudaStream_t stream) {
  dim3 grid((p.T + kRun - 1) / kRun, (2 * p.G + p.H + 3) / 4);
  const int es = sizeof(T), C = 2 * p.G * p.D + p.H * p.DV;
  const bool vec = p.D % 4 == 0 && p.DV % 4 == 0 && p.ld % 4 == 0 && C % 4 == 0 && al(p.x, 4 * es) && al(p.ring, 4 * es) &&
                   al(p.conv, 16) && al(p.qk, 16) && al(p.v, 16);
  const int m = p.D > p.DV ? p.D : p.DV;
  if (vec && m <= 128 && p.taps <= 4) prepare_kernel<T, 4, 1, true><<<grid, 128, 0, stream>>>(p);
  else if (vec) prepare_kernel<T, 4, 4, false><<<grid, 128, 0, stream>>>(p);
  else prepare_kernel<T, 1, 16, false><<<grid, 128, 0, stream>>>(p);
  return fail("prepare");
}

template <typename T>
int decays(const Args& p, cudaStream_t stream) {
  const bool vec = p.by_channel && p.D % 4 == 0 && p.ld_a % 4 == 0 && al(p.a, 4 * sizeof(T)) && al(p.dt_bias, 16) && al(p.g, 16);
  const long long n = (long long)p.T * p.H * (p.by_channel ? p.D / (vec ? 4 : 1) : 1);
  long long blocks = (n + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  if (vec) decay_kernel<T, 4><<<(unsigned)blocks, 256, 0, stream>>>(p);
  else decay_kernel<T, 1><<<(unsigned)blocks, 256, 0, stream>>>(p);
  return fail("decays");
}

template <typename T, int R, int L, int C, bool CH>
int scan_one(const Args& p, int vec, cudaStream_t stream) {
  using S = ScanShape<R, L, C, CH>;
  auto kern = scan_kernel<T, R, L, C, CH>;
  constexpr int smem = 2 * S::kStage * (int)sizeof(float);
  static_assert(smem <= 227 * 1024, "shared memory budget exceeded");
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) {
      mfb_host::set_error("delta_rule: cannot raise the shared memory limit");
      return 10;
    }
    set = true;
  }
  dim3 grid((p.DV + S::kCols - 1) / S::kCols, p.H, p.B);
  kern<<<grid, kScanThreads, smem, stream>>>(p, vec);
  return fail("scan");
}

template <typename T, bool CH>
int scan(const Args& p, cudaStream_t stream) {
  const int vec = p.D % 4 == 0 && p.DV % 4 == 0 && al(p.qk, 16) && al(p.v, 16) && al(p.g, 16) ? 1 : 0;
  if (p.D <= 32) return scan_one<T, 8, 4, 4, CH>(p, vec, stream);
  if (p.D <= 64) return scan_one<T, 8, 8, 4, CH>(p, vec, stream);
  if (p.D <= 128) {
    // few sequences and heads: half as many columns per CTA give twice as many CTAs
    if ((long long)p.B * p.H * ((p.DV + 63) / 64) <= 148) return scan_one<T, 8, 16, 4, CH>(p, vec, stream);
    return scan_one<T, 16, 8, 4, CH>(p, vec, stream);
  }
  if (p.D <= 256) return scan_one<T, 16, 16, 4, CH>(p, vec, stream);
  return scan_one<T, 16, 32, 4, CH>(p, vec, stream);
}

template <typename T>
int gate_out(const Args& p, cudaStream_t stream) {
  const long long items = (long long)p.T * p.H;
  const unsigned grid = (unsigned)((items + 3) / 4);
  const int es = sizeof(T);
  const bool vec = p.DV % 4 == 0 && p.ld_gate % 4 == 0 && p.ld_out % 4 == 0 && al(p.o, 16) && al(p.norm, 16) &&
                   al(p.gate, 4 * es) && al(p.out, 4 * es);
  if (vec) {
    if (p.DV <= 128) gate_out_kernel<T, 4, 1><<<grid, 128, 0, stream>>>(p);
    else gate_out_kernel<T, 4, 4><<<grid, 128, 0, stream>>>(p);
  } else {
    if (p.DV <= 128) gate_out_kernel<T, 1, 4><<<grid, 128, 0, stream>>>(p);
    else gate_out_kernel<T, 1, 16><<<grid, 128, 0, stream>>>(p);
  }
  return fail("gate_out");
}

int tx_log2_of(int DV) {
  int l = 0;
  while ((4 << l) < DV) ++l;
  return l;
}

template <typename T, int NT, int NR, int NI>
int decode_one(const Args& p, cudaStream_t stream) {
  const int l = tx_log2_of(p.DV);
  const size_t smem = (size_t)(3 * p.D + 2 * p.DV + NT / 32 + 2 * NT * 4) * sizeof(float) + 16;
  const bool fast = p.taps <= 4 && 2 * p.D + p.DV <= NI * NT && p.D <= NT && p.DV <= NT;
  if (fast) delta_decode_kernel<T, NT, NR, NI, true><<<dim3(p.H, p.B), NT, smem, stream>>>(p, l);
  else delta_decode_kernel<T, NT, NR, NI, false><<<dim3(p.H, p.B), NT, smem, stream>>>(p, l);
  return fail("decode");
}

// rows per thread with nt threads
int decode_rows(int D, int DV, int nt) {
  const int ty = nt >> tx_log2_of(DV);
  return ty < 1 ? 1 << 20 : (D + ty - 1) / ty;
}

template <typename T>
int decode(const Args& p, cudaStream_t stream) {
  const int n256 = decode_rows(p.D, p.DV, 256);
  if (n256 <= 4 && decode_rows(p.D, p.DV, 128) <= 8) return decode_one<T, 128, 8, 2>(p, stream);
  if (n256 <= 8) return decode_one<T, 256, 8, 2>(p, stream);
  if (n256 <= 16) return decode_one<T, 256, 16, 2>(p, stream);
  return decode_one<T, 512, 16, 2>(p, stream);
}

int check(const Args& p) {
  if (p.T < 0 || p.B < 1 || p.H < 1 || p.G < 1 || p.H % p.G || p.D < 1 || p.DV < 1 || p.D > 512 || p.DV > 512 || p.taps < 1 ||
      p.H > 65535 || p.B > 65535) {
    mfb_host::set_error("delta_rule: T=%d B=%d H=%d G=%d D=%d DV=%d taps=%d", p.T, p.B, p.H, p.G, p.D, p.DV, p.taps);
    return 1;
  }
  return 0;
}

}  // namespace dlt
}  // namespace mfb

extern "C" {
using namespace mfb;

// 1 when a decode step runs in one kernel (else it runs as portions of one row)
int mfb_delta_decode_supported(int D, int DV) {
  return DV % 4 == 0 && D <= 512 && DV <= 512 && dlt::decode_rows(D, DV, 512) <= 16 ? 1 : 0;
}

// floats of scratch for T rows
long long mfb_delta_scratch_floats(int T, int H, int G, int D, int DV, int by_channel) {
  auto up = [](long long n) { return (n + 3) / 4 * 4; };
  return up((long long)T * G * 2 * D) + 2 * up((long long)T * H * DV) + up((long long)T * H) + up((long long)T * H * (by_channel ? D : 1));
}

// The whole mixer core (see the file header). f32: the activations (x, b, a, gate, ring, out) are fp32, else bf16. cu_q null: a
// decode step of B rows, idle where slots < 0. scratch: mfb_delta_scratch_floats (portions only, 16-byte aligned).
int mfb_delta_rule(const void* x, long long ld, const void* b, const void* a, long long ld_a, const void* gate, long long ld_gate,
                   const float* conv, const float* a_log, const float* dt_bias, const float* norm, void* ring, float* state,
                   const int* cu_q, const int* context_lens, const int* slots, float* scratch, void* out, long long ld_out,
                   int T, int B, int H, int G, int D, int DV, int taps, int by_channel, int gate_silu, float eps, float out_scale,
                   int f32, cudaStream_t stream) {
  dlt::Args p;
  p.x = x; p.ld = ld; p.b = b; p.a = a; p.ld_a = ld_a; p.gate = gate; p.ld_gate = ld_gate; p.conv = conv; p.a_log = a_log;
  p.dt_bias = dt_bias; p.norm = norm; p.ring = ring; p.state = state; p.cu_q = cu_q; p.context_lens = context_lens;
  p.slots = slots; p.out = out; p.ld_out = ld_out; p.T = T; p.B = B; p.H = H; p.G = G; p.D = D; p.DV = DV; p.taps = taps;
  p.by_channel = by_channel; p.gate_silu = gate_silu; p.eps = eps; p.out_scale = out_scale;
  if (dlt::check(p)) return 1;
  if (T == 0) return 0;
  if (!cu_q) {
    if (!mfb_delta_decode_supported(D, DV) || T != B || !dlt::al(state, 16)) {
      mfb_host::set_error("delta_rule: decode step of %d rows, %d slots, D=%d DV=%d", T, B, D, DV);
      return 1;
    }
    return f32 ? dlt::decode<float>(p, stream) : dlt::decode<__nv_bfloat16>(p, stream);
  }
  auto up = [](long long n) { return (n + 3) / 4 * 4; };
  p.qk = scratch;
  p.v = p.qk + up((long long)T * G * 2 * D);
  p.o = p.v + up((long long)T * H * DV);
  p.beta = p.o + up((long long)T * H * DV);
  p.g = p.beta + up((long long)T * H);
  int rc = f32 ? dlt::prepare<float>(p, stream) : dlt::prepare<__nv_bfloat16>(p, stream);
  if (!rc) rc = f32 ? dlt::decays<float>(p, stream) : dlt::decays<__nv_bfloat16>(p, stream);
  if (rc) return rc;
  if (f32) rc = by_channel ? dlt::scan<float, true>(p, stream) : dlt::scan<float, false>(p, stream);
  else rc = by_channel ? dlt::scan<__nv_bfloat16, true>(p, stream) : dlt::scan<__nv_bfloat16, false>(p, stream);
  if (rc) return rc;
  return f32 ? dlt::gate_out<float>(p, stream) : dlt::gate_out<__nv_bfloat16>(p, stream);
}

}  // extern "C"
