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
//   gates_kernel, chunk_kernel: portions of 16-bit models in chunks of 64 tokens on the tensor cores (see there)
//   scan_kernel:   portions of 32-bit models and of other sizes, token by token on the FMA pipes; a CTA holds 32 columns of one
//                  head's S in registers
//   finish_kernel: norm, gate and the new n and m of a portion (which other CTAs read until then)
//   decode_kernel: one row per slot, all in one pass; rows of idle slots (slot_mapping < 0) become zeros
#include "mma_sync.cuh"

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
  float* gates;              // [H, T, 6] of the chunks
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

// ---- portions in chunks of 64 tokens ----------------------------------------------------------------------------------------
// Within a chunk that starts from (S, n, m0), with b_t the sum of the log forget gates up to t and a_s = i_s - b_s:
//   A_t = max(m0, max_{s <= t} a_s),  m_t = b_t + A_t
//   o_t (max(|q . n_t|, e^-m_t) + 1e-6) = e^(m0 - A_t) S^T q_t + sum_{s <= t} (q_t . k_s) e^(a_s - A_t) v_s,   q . n_t likewise
//   after the last token: S <- e^(m0 - A) S + sum_s k_s (e^(a_s - A) v_s)^T, n likewise, m <- b + A
// so that every exponent is at most zero. a, its running maximum and b do not depend on what came before the chunk: gates_kernel
// works them out for all chunks at once, in fp64, as pairs of fp32 numbers (their differences stay exact where the sums are
// large). chunk_kernel walks over the chunks of one head: four warps hold 16 columns of S each, transposed, as fp32 MMA
// accumulators. q, k and v enter the products as they are (bf16); fp32 factors enter as sums of bf16 numbers: two for S and the
// weights in the read-out, three for the weighted values that go into S, whose error would stay.
constexpr int kChunk = 64;

// a warp per head, two tokens per lane
template <typename T>
__global__ void __launch_bounds__(256) gates_kernel(const Args a) {
  extern __shared__ float sh[];                      // [64][2 H] gate inputs
  const int b = blockIdx.y, r0 = a.cu_q[b], rows = a.cu_q[b + 1] - r0, t0 = blockIdx.x * kChunk;
  if (t0 >= rows) return;
  const int n = min(kChunk, rows - t0), H = a.H;
  for (int i = threadIdx.x; i < n * 2 * H; i += blockDim.x) {
    const int t = i / (2 * H), c = i % (2 * H);
    sh[i] = ld(reinterpret_cast<const T*>(a.proj) + (long long)(r0 + t0 + t) * a.ld + a.col_i() + c);
  }
  __syncthreads();
  const int lane = threadIdx.x & 31;
  for (int h = threadIdx.x >> 5; h < H; h += blockDim.x >> 5) {
    double i_[2], f[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = 2 * lane + e;
      i_[e] = t < n ? input_gate(sh[t * 2 * H + h] + a.bi[h], a.cap) : -INFINITY;
      f[e] = t < n ? forget_gate(sh[t * 2 * H + H + h] + a.bf[h], a.cap) : 0.f;
    }
    double sum = f[0] + f[1];
#pragma unroll
    for (int o = 1; o < 32; o *= 2) {
      const double up = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += up;
    }
    const double b1 = sum, b0 = sum - f[1];
    const double a0 = i_[0] - b0, a1 = i_[1] - b1;
    double top = fmax(a0, a1);
#pragma unroll
    for (int o = 1; o < 32; o *= 2) {
      const double up = __shfl_up_sync(0xffffffffu, top, o);
      if (lane >= o) top = fmax(top, up);
    }
    const double before = __shfl_up_sync(0xffffffffu, top, 1);
    const double c0 = lane ? fmax(before, a0) : a0;
    float* g = a.gates + ((long long)h * a.T + r0 + t0 + 2 * lane) * 6;
    auto put = [](float* p, double x) {
      const float hi = static_cast<float>(x);
      p[0] = hi;
      p[1] = static_cast<float>(x - hi);
    };
    if (2 * lane < n) { put(g, a0); put(g + 2, c0); put(g + 4, b0); }
    if (2 * lane + 1 < n) { put(g + 6, a1); put(g + 8, top); put(g + 10, b1); }
  }
}

// DP: padded key size; STAGES: buffers of q, k and v
template <int DP, int STAGES>
struct ChunkShape {
  static constexpr int kQPitch = DP * 2 + 16, kVPitch = 64 * 2 + 16;      // bytes; rows shift by a bank group
  static constexpr int kQBytes = kChunk * kQPitch, kVBytes = kChunk * kVPitch;
  static constexpr int kStage = 2 * kQBytes + kVBytes + kChunk * 6 * 4;
  static constexpr int kSmem = STAGES * kStage + 2 * kVBytes + DP * 4 + 3 * kChunk * 4;
};

template <int DP, int STAGES>
__global__ void __launch_bounds__(128, 2) chunk_kernel(const Args p) {
  using Sh = ChunkShape<DP, STAGES>;
  constexpr int KS = DP / 16, NT = DP / 8;
  extern __shared__ __align__(16) uint8_t smem[];
  const int b = blockIdx.z, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int r0 = p.cu_q[b], rows = p.cu_q[b + 1] - r0;
  if (rows <= 0) return;
  const int start = p.context_lens[b] - rows, D = p.D, DV = p.DV, H = p.H;
  const int slice = blockIdx.x * 64, dv0 = slice + warp * 16;
  const int g = lane >> 2, tq = lane & 3;
  uint8_t* sP = smem + STAGES * Sh::kStage;           // weights: high, low
  float* sN = reinterpret_cast<float*>(sP + 2 * Sh::kVBytes);
  float* sScale = sN + DP;                            // e^(m0 - A_t)
  float* sInv = sScale + kChunk;                      // q scale / normaliser
  float* sW = sInv + kChunk;                          // weight of a token in the state after the chunk
  const long long head = (long long)b * H + h;
  const __nv_bfloat16* base = reinterpret_cast<const __nv_bfloat16*>(p.proj) + (long long)r0 * p.ld;

  float s[NT][4];                                     // S^T: rows dv0 + g, dv0 + g + 8; columns 8 j + 2 tq, + 1
  {
    const float* S = p.S + head * D * DV;
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = 8 * j + 2 * tq + (e & 1), v = dv0 + g + (e >> 1) * 8;
        s[j][e] = (start > 0 && d < D && v < DV) ? S[(long long)d * DV + v] : 0.f;
      }
  }
  for (int d = tid; d < DP; d += 128) sN[d] = (start > 0 && d < D) ? p.n[head * D + d] : 0.f;
  float m0 = start > 0 ? p.m[head] : 0.f;

  const int chunks = (rows + kChunk - 1) / kChunk;
  auto fetch = [&](int c) {
    uint8_t* st = smem + (c % STAGES) * Sh::kStage;
    const uint32_t sq = smem_u32(st);
    const int n = min(kChunk, rows - c * kChunk);
    for (int i = tid; i < kChunk * (DP / 8); i += 128) {
      const int t = i / (DP / 8), d = (i % (DP / 8)) * 8;
      const bool in = t < n && d < D;
      const __nv_bfloat16* src = base + (long long)(c * kChunk + (in ? t : 0)) * p.ld + h * D + (in ? d : 0);
      cp16(sq + t * Sh::kQPitch + d * 2, src, in ? 16 : 0);
      cp16(sq + Sh::kQBytes + t * Sh::kQPitch + d * 2, src + p.col_k(), in ? 16 : 0);
    }
    for (int i = tid; i < kChunk * 8; i += 128) {
      const int t = i / 8, v = (i % 8) * 8;
      const bool in = t < n && slice + v < DV;
      const __nv_bfloat16* src = base + (long long)(c * kChunk + (in ? t : 0)) * p.ld + p.col_v() + h * DV + (in ? slice + v : 0);
      cp16(sq + 2 * Sh::kQBytes + t * Sh::kVPitch + v * 2, src, in ? 16 : 0);
    }
    // gates of padding tokens: weight zero; their maximum and sum are not used
    float* sg = reinterpret_cast<float*>(st + 2 * Sh::kQBytes + Sh::kVBytes);
    const float* src = p.gates + ((long long)h * p.T + r0 + c * kChunk) * 6;
    for (int i = tid; i < kChunk * 6; i += 128) sg[i] = i < n * 6 ? src[i] : (i % 6 == 0 ? -INFINITY : 0.f);
    cp_commit();
  };
  fetch(0);
  for (int c = 0; c < chunks; ++c) {
    const int n = min(kChunk, rows - c * kChunk);
    if (STAGES > 1 && c + 1 < chunks) { fetch(c + 1); cp_wait<1>(); }
    else cp_wait<0>();
    __syncthreads();
    uint8_t* st = smem + (c % STAGES) * Sh::kStage;
    const uint32_t sq = smem_u32(st), sk = sq + Sh::kQBytes, sv = sk + Sh::kQBytes, sp = smem_u32(sP);
    const float* sg = reinterpret_cast<const float*>(st + 2 * Sh::kQBytes + Sh::kVBytes);
    const float* gl = sg + (n - 1) * 6;
    const bool old_top = m0 > gl[2];                  // A after the last token
    const float eh = old_top ? m0 : gl[2], el = old_top ? 0.f : gl[3];
    const float keep = old_top ? 1.f : __expf((m0 - eh) - el);
    if (tid < kChunk) sW[tid] = __expf((sg[tid * 6] - eh) + (sg[tid * 6 + 1] - el));
    // ---- scores of the warp's 16 tokens, their weights and sums ----
    {
      float acc[8][4] = {}, nq[4] = {};
      const int last = 2 * warp + 1;                  // key tiles up to the diagonal
#pragma unroll
      for (int k = 0; k < KS; ++k) {
        uint32_t qa[4];
        ldsm4(qa, sq + (warp * 16 + (lane & 15)) * Sh::kQPitch + k * 32 + (lane >> 4) * 16);
#pragma unroll
        for (int j = 0; j < 8; j += 2)
          if (j <= last) {
            uint32_t kb[4];                           // tiles j and j + 1, both halves of the 16 dimensions
            ldsm4(kb, sk + (j * 8 + (lane & 7) + (lane >> 4) * 8) * Sh::kQPitch + k * 32 + ((lane >> 3) & 1) * 16);
            mma(acc[j], qa, kb[0], kb[1]);
            mma(acc[j + 1], qa, kb[2], kb[3]);
          }
        // n as the first column of a tile
        float x0 = g == 0 ? sN[k * 16 + 2 * tq] : 0.f, x1 = g == 0 ? sN[k * 16 + 2 * tq + 1] : 0.f;
        float y0 = g == 0 ? sN[k * 16 + 8 + 2 * tq] : 0.f, y1 = g == 0 ? sN[k * 16 + 9 + 2 * tq] : 0.f;
#pragma unroll
        for (int e = 0; e < 3; ++e) {
          const uint32_t b0 = take_bf16(x0, x1), b1 = take_bf16(y0, y1);
          mma(nq, qa, b0, b1);
        }
      }
      float sum[2] = {0.f, 0.f}, ah[2], al[2], scale[2], floor_[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const float* gt = sg + min(warp * 16 + g + 8 * r, n - 1) * 6;
        const bool own = m0 > gt[2];
        ah[r] = own ? m0 : gt[2];
        al[r] = own ? 0.f : gt[3];
        scale[r] = own ? 1.f : __expf((m0 - ah[r]) - al[r]);
        floor_[r] = __expf(-((gt[4] + ah[r]) + (gt[5] + al[r])));
      }
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (j <= last) {
          const int s0 = j * 8 + 2 * tq;
          const float h0 = sg[s0 * 6], l0 = sg[s0 * 6 + 1], h1 = sg[s0 * 6 + 6], l1 = sg[s0 * 6 + 7];
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            const int t = warp * 16 + g + 8 * r;
            float w0 = s0 <= t ? acc[j][2 * r] * __expf((h0 - ah[r]) + (l0 - al[r])) : 0.f;
            float w1 = s0 + 1 <= t ? acc[j][2 * r + 1] * __expf((h1 - ah[r]) + (l1 - al[r])) : 0.f;
            sum[r] += w0 + w1;
            uint8_t* dst = sP + t * Sh::kVPitch + s0 * 2;
            *reinterpret_cast<uint32_t*>(dst) = take_bf16(w0, w1);
            *reinterpret_cast<uint32_t*>(dst + Sh::kVBytes) = take_bf16(w0, w1);
          }
        }
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 1);
        sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 2);
        if (tq == 0) {                                // column 0 of the tile with n lies in this lane
          const int t = warp * 16 + g + 8 * r;
          const float d = fmaf(scale[r], nq[2 * r], sum[r]) * p.q_scale;
          sScale[t] = scale[r];
          sInv[t] = p.q_scale / (fmaxf(fabsf(d), floor_[r]) + 1e-6f);
        }
      }
    }
    __syncthreads();
    // ---- read-out of the warp's 16 columns for all tokens ----
    if (dv0 < DV) {
      float o[4][2][4] = {};
#pragma unroll
      for (int k = 0; k < KS; ++k) {
        uint32_t hi[4], lo[4];                        // S as a K x N operand: columns dv0.. (0, 1), dv0 + 8.. (2, 3)
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
          uint32_t qa[4];
          ldsm4(qa, sq + (m * 16 + (lane & 15)) * Sh::kQPitch + k * 32 + (lane >> 4) * 16);
          mma(o[m][0], qa, hi[0], hi[1]);
          mma(o[m][1], qa, hi[2], hi[3]);
          mma(o[m][0], qa, lo[0], lo[1]);
          mma(o[m][1], qa, lo[2], lo[3]);
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
        uint32_t vb[4];                               // tokens 16 k.. of columns dv0.. (0, 1), dv0 + 8.. (2, 3)
        ldsm4t(vb, sv + (k * 16 + (lane & 15)) * Sh::kVPitch + warp * 32 + (lane >> 4) * 16);
#pragma unroll
        for (int m = k; m < 4; ++m) {
          const uint32_t at = sp + (m * 16 + (lane & 15)) * Sh::kVPitch + k * 32 + (lane >> 4) * 16;
          uint32_t wa[4];
          ldsm4(wa, at);
          mma(o[m][0], wa, vb[0], vb[1]);
          mma(o[m][1], wa, vb[2], vb[3]);
          ldsm4(wa, at + Sh::kVBytes);
          mma(o[m][0], wa, vb[0], vb[1]);
          mma(o[m][1], wa, vb[2], vb[3]);
        }
      }
#pragma unroll
      for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int t = m * 16 + g + 8 * r;
          if (t >= n) continue;
          const float inv = sInv[t];
          float* dst = p.o + ((long long)(r0 + c * kChunk + t) * H + h) * DV + dv0 + 2 * tq;
#pragma unroll
          for (int j = 0; j < 2; ++j)
            if (dv0 + j * 8 + 2 * tq < DV)
              *reinterpret_cast<float2*>(dst + j * 8) = make_float2(o[m][j][2 * r] * inv, o[m][j][2 * r + 1] * inv);
        }
    }
    // ---- state after the chunk ----
    if (dv0 < DV) {
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[j][e] *= keep;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        uint32_t va[4], w1[4], w2[4], w3[4];          // V^T: rows dv0 + g (0, 2), + 8 (1, 3); tokens 16 k + 2 tq (0, 1), + 8 (2, 3)
        ldsm4t(va, sv + (k * 16 + (lane & 7) + (lane >> 4) * 8) * Sh::kVPitch + warp * 32 + ((lane >> 3) & 1) * 16);
#pragma unroll
        for (int q = 0; q < 2; ++q) {
          const int t = k * 16 + 2 * tq + 8 * q;
          const float x = sW[t], y = sW[t + 1];
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&va[2 * q + r]));
            float f0 = f.x * x, f1 = f.y * y;
            w1[2 * q + r] = take_bf16(f0, f1);
            w2[2 * q + r] = take_bf16(f0, f1);
            w3[2 * q + r] = take_bf16(f0, f1);
          }
        }
#pragma unroll
        for (int j = 0; j < NT; j += 2) {
          uint32_t kb[4];                             // tokens 16 k.. of dimensions 8 j.. (0, 1), 8 j + 8.. (2, 3)
          ldsm4t(kb, sk + (k * 16 + (lane & 15)) * Sh::kQPitch + j * 16 + (lane >> 4) * 16);
          mma(s[j], w1, kb[0], kb[1]);
          mma(s[j + 1], w1, kb[2], kb[3]);
          mma(s[j], w2, kb[0], kb[1]);
          mma(s[j + 1], w2, kb[2], kb[3]);
          mma(s[j], w3, kb[0], kb[1]);
          mma(s[j + 1], w3, kb[2], kb[3]);
        }
      }
    }
    for (int d = tid; d < DP; d += 128) {
      float x = sN[d] * keep;
      const uint8_t* kcol = st + Sh::kQBytes + d * 2;
#pragma unroll 8
      for (int t = 0; t < kChunk; ++t)
        x = fmaf(sW[t], __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(kcol + t * Sh::kQPitch)), x);
      sN[d] = x;
    }
    m0 = (gl[4] + eh) + (gl[5] + el);
    __syncthreads();
    if (STAGES == 1 && c + 1 < chunks) fetch(c + 1);
  }
  float* S = p.S + head * D * DV;
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = 8 * j + 2 * tq + (e & 1), v = dv0 + g + (e >> 1) * 8;
      if (d < D && v < DV) S[(long long)d * DV + v] = s[j][e];
    }
  if (blockIdx.x == 0) {
    for (int d = tid; d < D; d += 128) p.n_new[head * D + d] = sN[d];
    if (tid == 0) p.m_new[head] = m0;
  }
}

bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

bool chunks_ok(const Args& a) {
  return a.D % 8 == 0 && a.DV % 8 == 0 && a.D <= 256 && a.ld % 8 == 0 && al16(a.proj) && al16(a.o) && a.H <= 64;
}

template <int DP, int STAGES>
int chunk_launch(const Args& a, cudaStream_t stream) {
  using Sh = ChunkShape<DP, STAGES>;
  static_assert(2 * (Sh::kSmem + 1024) <= 233472, "two CTAs per SM");
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(chunk_kernel<DP, STAGES>, cudaFuncAttributeMaxDynamicSharedMemorySize, Sh::kSmem) != cudaSuccess) {
      mfb_host::set_error("matrix_memory: cannot raise the shared memory limit");
      return 10;
    }
    attr_set = true;
  }
  chunk_kernel<DP, STAGES><<<dim3((a.DV + 63) / 64, a.H, a.B), 128, Sh::kSmem, stream>>>(a);
  return 0;
}

int in_chunks(const Args& a, int longest, cudaStream_t stream) {
  gates_kernel<__nv_bfloat16><<<dim3((longest + kChunk - 1) / kChunk, a.B), 256, (size_t)kChunk * 2 * a.H * 4, stream>>>(a);
  int rc;
  if (a.D <= 32) rc = chunk_launch<32, 2>(a, stream);
  else if (a.D <= 64) rc = chunk_launch<64, 2>(a, stream);
  else if (a.D <= 128) rc = chunk_launch<128, 2>(a, stream);
  else rc = chunk_launch<256, 1>(a, stream);
  if (rc) return rc;
  const long long items = (long long)a.T * a.H + (long long)a.B * a.H;
  finish_kernel<__nv_bfloat16><<<(unsigned)((items + 3) / 4), 128, 0, stream>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : 2;
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
  return (long long)T * H * (DV + 6) + (long long)B * H * (D + 1) + 4;
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
  mmem::Args a;
  a.proj = proj; a.ld = ld; a.bi = bi; a.bf = bf; a.norm = norm; a.S = S; a.n = n; a.m = m; a.cu_q = cu_q;
  a.context_lens = context_lens; a.slots = slots; a.out = out;
  a.o = scratch; a.n_new = scratch + (long long)T * H * DV; a.m_new = a.n_new + (long long)B * H * D;
  a.gates = a.m_new + (long long)B * H;
  a.T = T; a.B = B; a.H = H; a.D = D; a.DV = DV; a.cap = cap; a.eps = eps; a.q_scale = 1.f / sqrtf((float)D);
  int rc;
  if (cu_q && !f32 && longest > 0 && mmem::chunks_ok(a)) rc = mmem::in_chunks(a, longest, stream);
  else if (cu_q) rc = f32 ? mmem::portions<float>(a, stream) : mmem::portions<__nv_bfloat16>(a, stream);
  else rc = f32 ? mmem::decode<float>(a, stream) : mmem::decode<__nv_bfloat16>(a, stream);
  if (rc == 2) mfb_host::set_error("matrix_memory: launch failed");
  return rc;
}

}  // extern "C"
