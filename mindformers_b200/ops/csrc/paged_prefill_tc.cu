// Prefill attention of a ragged batch over a paged bf16 cache on the tensor cores (sm_100a, tcgen05 + TMA), grouped-query
// attention with query / key size up to 192 and value size up to 128 (multiples of 8), optional chunked mask and softmax sink.
//
// Sequence b brings the rows cu_q[b] .. cu_q[b + 1] - 1 of q; its keys and values, those rows included, are in the cache
// already, so a whole prompt, a later portion of a prompt and any mix of sequences are the same problem: row r of the
// portion sits at position context_lens[b] - q_len + r and sees keys up to itself, with `chunk` > 0 only those of its
// own chunk of `chunk` positions (counted from position 0). `sink` [Hq] adds exp(sink_h) to the denominator. A soft cap
// bounds the scores (cap * tanh(score / cap)).
//
// The tensor-core pipeline is the one of flash_attention_fwd2.cu (P goes back into tensor memory and is read from there
// by the P V product), with one 128-row query tile per CTA and one stage of K and of V: a CTA then takes half of an SM's
// tensor memory and at most half of its shared memory, and two of them share an SM: while one waits for its products or
// its softmax the other works. K of the next key tile loads during the softmax of this one, V during the scores and the
// softmax, so one stage of each is enough. A CTA's roles run through all of its tiles (see the launcher): the
// loads and the first scores of a tile run under the last softmax and the output of the one before, which is what counts
// when a tile sees few keys (chunks, short portions). What else differs:
//   - a sliding window (`window` > 0) hides the keys that lie `window` or more positions before the row;
//   - with `all_values` every query head's weights are applied to the values of every key / value head: by a kernel of its own
//     (below), with a sink or a soft cap as items of their own;
//   - rows of K and V may lie further apart than their heads fill (slices of one product);
//   - work comes as a list of (sequence, first row of q, rows, position of the first row), one entry per query tile; only
//     key tiles that some row of the tile sees are visited, from the chunk of its first row to its last row;
//   - K / V tiles (128 consecutive positions) are assembled from the sequence's pages, one TMA box per page and 64
//     columns; pages past the end of the sequence repeat the tile's first page and are masked;
//   - head sizes are padded to 64, 128 or 192 columns (192: one CTA per SM): q is read through a three-dimensional map that fills the columns past
//     the head with zeros, so whatever a K box holds there does not count; columns of V past the head reach only
//     columns of the result that are not stored;
//   - the result is written row by row: a portion may end anywhere.
//
// Roles (192 threads): warp 0 TMA producer, warp 1 MMA issuer + TMEM owner, warps 2..5 softmax. Every wait is bounded (common.cuh).
#include <type_traits>

#include "common.cuh"

namespace mfb {
namespace ppt {

constexpr int kThreads = 192;
constexpr int kTile = 128;
constexpr int kSubBytes = kTile * 128;     // [128 rows][128 B] swizzled sub-tile (64 bf16 columns)
constexpr float kRescaleThreshold = 8.0f;  // log2 units

struct Args {
  const int4* work;          // [n_work]: sequence, first row of q, rows, position of the first row
  int n_items;               // n_work x query heads x vheads, in this order
  const int* block_tables;   // [B, max_blocks]
  const float* sink;         // [Hq] or null
  __nv_bfloat16* out;        // [T, Hq, vheads, DV]
  int num_q_heads, group, D, DV, block_size, max_blocks, chunk, window;
  int vheads;                // value heads per query head: 1 (its own) or all
  float scale_log2;
  float cap_log2, cap_scale;   // soft cap of the scores in log2 units (CAP kernels) and scale / cap
  float cap_poly[5];           // capped score (log2 units) = s * polynomial in s^2, for |s| * cap_scale <= kPolyReach
  long long ld_out;
  float out_scale;
  int* status;
};

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// cap * tanh(x) from exp(2 |x|): the error stays at a few 1e-7 of the cap
__device__ __forceinline__ float capped(float x, float cap) {
  const float e = ex2(fabsf(x) * 2.8853900817779268f);
  float r;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(e + 1.f));
  return copysignf(cap * fmaf(-2.f, r, 1.f), x);
}
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
__device__ __forceinline__ uint64_t add2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ float fmax3(float a, float b, float c) {
  float d;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
  return d;
}
__device__ __forceinline__ void tmem_st_32x32b_x32(uint32_t taddr, const uint32_t* r) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16,"
      " %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};\n"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
        "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]),
        "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]),
        "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
      : "memory");
}

// tanh(x) / x as a polynomial in x^2 on |x| <= kPolyReach (Chebyshev interpolation of degree 4 on [0, kPolyReach^2]: relative
// error 7.4e-8). It runs on the FMA pipes two scores at a time, which leaves the exponentials to the softmax; the launcher
// folds the scales into the coefficients.
constexpr float kPolyReach = 0.6f;
constexpr float kTanhRatio[5] = {0.999999926f, -0.33332302f, 0.133100644f, -0.0520966534f, 0.0154687513f};

// HQ: padded query / key size (64, 128 or 192), HV: padded value size (64 or 128); CAP: scores are soft-capped
template <int HQ, int HV, bool CAP>
__global__ void __launch_bounds__(kThreads, HQ > 128 ? 1 : 2)
paged_prefill_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                        const __grid_constant__ CUtensorMap tmV, const Args args) {
  constexpr int QB = HQ / 64, VB = HV / 64;          // 64-column sub-tiles
  constexpr int kQBytes = QB * kSubBytes, kVBytes = VB * kSubBytes;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) &
                                             ~static_cast<uintptr_t>(1023));
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + kQBytes;
  uint8_t* sV = sK + kQBytes;
  uint8_t* sOut = sV + kVBytes;               // 2 KB per softmax warp
  uint64_t* bars = reinterpret_cast<uint64_t*>(sOut + 4 * 2048);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;
  uint64_t* k_empty = bars + 2;
  uint64_t* v_full = bars + 3;
  uint64_t* v_empty = bars + 4;
  uint64_t* s_full = bars + 5;      // S complete
  uint64_t* p_ready = bars + 6;     // P written (128 arrivals)
  uint64_t* pv_done = bars + 7;     // P V complete
  uint64_t* q_empty = bars + 8;     // last scores of a query tile complete
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(bars + 9);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_holder + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  struct Tile { int b, head, vsel, q0, rows, pos0, lo, n_kv; };      // key tiles lo .. n_kv - 1
  auto first_of = [&](int pos) {            // first position that `pos` sees; does not fall as pos grows
    int lo = args.chunk > 0 ? pos - pos % args.chunk : 0;
    if (args.window > 0 && pos - args.window + 1 > lo) lo = pos - args.window + 1;
    return lo;
  };
  auto tile_of = [&](int item) {
    Tile t;
    t.vsel = item % args.vheads;
    item /= args.vheads;
    const int4 w = args.work[item / args.num_q_heads];
    t.head = item % args.num_q_heads;
    t.b = w.x; t.q0 = w.y; t.rows = w.z; t.pos0 = w.w;
    t.lo = first_of(t.pos0) / kTile;
    t.n_kv = (t.pos0 + t.rows - 1) / kTile + 1;
    return t;
  };
  const int first_item = static_cast<int>(blockIdx.x), step = static_cast<int>(gridDim.x);

  if (threadIdx.x == 0) {
    *abort_flag = 0;
    for (int i = 0; i < 9; ++i) mbar_init(smem_u32(&bars[i]), &bars[i] == p_ready ? 128 : 1);
    fence_barrier_init();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_holder), 256);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_holder;
  const uint32_t tmem_S = tmem_base, tmem_O = tmem_base + kTile;   // P lives in the first 64 columns of S
  if (warp == 0) {
    // ------------------------------ TMA producer (the whole warp, one lane issues) ------------------------------
    const bool leader = elect_one();
    const int bs = args.block_size;
    uint32_t it = 0, n = 0;                          // key tiles and query tiles so far
    bool ok = true;
    // wait until a buffer is free (the lanes agree on the outcome) and announce what goes there
    auto claim = [&](uint64_t* empty, uint32_t parity, uint64_t* full, uint32_t bytes) {
      ok = mbar_wait(smem_u32(empty), parity, abort_flag, args.status, kStatusWaitTimeoutProducer);
      ok = __all_sync(0xffffffffu, ok);
      if (ok && leader) mbar_expect_tx(smem_u32(full), bytes);
      __syncwarp();
    };
    for (int item = first_item; item < args.n_items && ok; item += step, ++n) {
      const Tile t = tile_of(item);
      const int* table = args.block_tables + static_cast<size_t>(t.b) * args.max_blocks;
      const int kv_head = t.head / args.group, end = t.pos0 + t.rows;
      const int kcol = kv_head * args.D, vcol = (args.vheads > 1 ? t.vsel : kv_head) * args.DV;
      int page = tile_page(table, bs, t.lo * kTile, end);
      claim(q_empty, (n & 1) ^ 1, q_full, kQBytes);
      if (!ok) break;
      if (leader)
        for (int c = 0; c < QB; ++c) tma_load_3d(smem_u32(sQ) + c * kSubBytes, &tmQ, smem_u32(q_full), c * 64, t.head, t.q0);
      __syncwarp();
      for (int j = t.lo; j < t.n_kv; ++j, ++it) {
        const uint32_t ph = it & 1;
        claim(k_empty, ph ^ 1, k_full, kQBytes);
        if (!ok) break;
        tma_load_pages(leader, smem_u32(sK), kSubBytes, &tmK, smem_u32(k_full), page, bs, kcol, QB);
        const int next = j + 1 < t.n_kv ? tile_page(table, bs, (j + 1) * kTile, end) : 0;
        claim(v_empty, ph ^ 1, v_full, kVBytes);
        if (!ok) break;
        tma_load_pages(leader, smem_u32(sV), kSubBytes, &tmV, smem_u32(v_full), page, bs, vcol, VB);
        page = next;
      }
    }
  } else if (warp == 1) {
    // ------------------------------ MMA issuer (the whole warp, one lane issues) ------------------------------
    constexpr uint32_t IDESC_QK = umma_idesc_bf16(kTile, kTile, 0, 0);  // A = Q K-major (smem), B = K K-major
    constexpr uint32_t IDESC_PV = umma_idesc_bf16(kTile, HV, 0, 1);     // A = P (tensor memory), B = V MN-major
    const bool leader = elect_one();
    const uint64_t q_desc = umma_desc_kmajor_sw128(smem_u32(sQ)), k_desc = umma_desc_kmajor_sw128(smem_u32(sK));
    const uint64_t v_desc = umma_desc_mnmajor_sw128(smem_u32(sV), kSubBytes);
    uint32_t it = 0, n = 0;
    bool ok = true, first_key = true;                // first_key: the pending P V product starts its query tile's sum
    auto wait = [&](uint64_t* bar, uint32_t parity) {
      ok = mbar_wait(smem_u32(bar), parity, abort_flag, args.status, kStatusWaitTimeoutMma);
      ok = __all_sync(0xffffffffu, ok);
    };
    // O (+)= P V of key tile it - 1
    auto issue_pv = [&]() {
      const uint32_t ph = (it - 1) & 1;
      wait(v_full, ph);
      if (ok) wait(p_ready, ph);
      if (!ok) return;
      tc_fence_after();
#pragma unroll
      for (int k = 0; k < kTile / 16; ++k)           // bf16 pairs: 8 columns of P per 16 keys
        umma_f16_ts_warp(leader, tmem_O, tmem_S + k * 8, v_desc + ((k * 16 * 128) >> 4), IDESC_PV, (!first_key || k > 0) ? 1u : 0u);
      umma_commit_warp(leader, smem_u32(pv_done));
      umma_commit_warp(leader, smem_u32(v_empty));
    };
    for (int item = first_item; item < args.n_items && ok; item += step, ++n) {
      const Tile t = tile_of(item);
      for (int j = t.lo; j < t.n_kv; ++j) {
        if (it > 0) issue_pv();
        if (ok && j == t.lo) wait(q_full, n & 1);
        // ---- S = Q K(j)^T: overwrites S / P, executes behind the P V product issued just above ----
        if (ok) wait(k_full, it & 1);
        if (!ok) break;
        tc_fence_after();
#pragma unroll
        for (int k = 0; k < HQ / 16; ++k) {
          constexpr int kSubUnits = kSubBytes >> 4;
          const int off = (k >> 2) * kSubUnits + (k & 3) * 2;
          umma_f16_ss_warp(leader, tmem_S, q_desc + off, k_desc + off, IDESC_QK, k > 0 ? 1u : 0u);
        }
        umma_commit_warp(leader, smem_u32(s_full));
        umma_commit_warp(leader, smem_u32(k_empty));
        if (j == t.n_kv - 1) umma_commit_warp(leader, smem_u32(q_empty));
        first_key = j == t.lo;
        ++it;
      }
    }
    if (ok && it > 0) issue_pv();
  } else {
    // ------------------------------ softmax warpgroup ------------------------------
    const int ew = warp & 3;                       // TMEM lane quarter of this warp
    const int row = ew * 32 + lane;
    const uint32_t lane_base = static_cast<uint32_t>(ew * 32) << 16;
    const uint32_t s_tmem = tmem_S + lane_base;
    const uint32_t o_tmem = tmem_O + lane_base;
    bool ok = true;
    const uint64_t scale2 = pack2(args.scale_log2, args.scale_log2);
    uint32_t it = 0;
    for (int item = first_item; item < args.n_items; item += step) {
      const Tile t = tile_of(item);
      const int lo = t.lo, n_kv = t.n_kv;
      const int my_pos = t.pos0 + row;
      const int my_first = first_of(my_pos);         // first key this row may see
      float m_used = -INFINITY, l_sum = 0.f;
      for (int j = lo; j < n_kv; ++j, ++it) {
        ok = mbar_wait(smem_u32(s_full), it & 1, abort_flag, args.status, kStatusWaitTimeoutEpilogue);
        if (!ok) break;
        tc_fence_after();
        // columns [col_lo, col_hi] of this key tile are visible to the row (none, if the range is empty)
        const int col_lo = my_first - j * kTile;
        const int col_hi = my_pos - j * kTile;
        // the bounds grow with the row: blocks of columns that every row of the warp sees need no mask, and halves that
        // no row sees no exponentials
        const int hi_min = __shfl_sync(0xffffffffu, col_hi, 0), hi_max = __shfl_sync(0xffffffffu, col_hi, 31);
        const int lo_min = __shfl_sync(0xffffffffu, col_lo, 0), lo_max = __shfl_sync(0xffffffffu, col_lo, 31);
        // the softmax of one key tile, compiled twice: tiles that every row of the warp sees whole carry no masking code
        auto softmax_tile = [&](auto mask_tag) {
          constexpr bool MASK = decltype(mask_tag)::value;
          // pass 1: row maximum (four independent chains of three-input maxima); the scores are not kept
          float mxs[4];
          {
            uint32_t sr[kTile];
#pragma unroll
            for (int c = 0; c < 4; ++c) {
              uint32_t (&r)[32] = *reinterpret_cast<uint32_t(*)[32]>(&sr[c * 32]);
              tmem_ld_32x32b_x32(s_tmem + c * 32, r);
            }
            tmem_ld_wait();
            float* s = reinterpret_cast<float*>(sr);
#pragma unroll
            for (int a = 0; a < 4; ++a) {
              if (MASK && hi_min < a * 32 + 31) {
#pragma unroll
                for (int i = a * 32; i < a * 32 + 32; ++i)
                  if (i > col_hi) s[i] = -INFINITY;
              }
              if (MASK && lo_max > a * 32) {
#pragma unroll
                for (int i = a * 32; i < a * 32 + 32; ++i)
                  if (i < col_lo) s[i] = -INFINITY;
              }
              float m = s[a * 32];
#pragma unroll
              for (int i = 1; i + 1 < 32; i += 2) m = fmax3(m, s[a * 32 + i], s[a * 32 + i + 1]);
              mxs[a] = fmaxf(m, s[a * 32 + 31]);
            }
          }
          float mx = fmaxf(fmaxf(mxs[0], mxs[1]), fmaxf(mxs[2], mxs[3]));
          if (!CAP) mx *= args.scale_log2;
          else if (mx != -INFINITY) mx = capped(mx * args.cap_scale, args.cap_log2);      // the cap keeps the order
          float alpha = 1.f;
          if (j == lo) {
            m_used = mx;                               // -inf when this row sees nothing in its tile's first key tile
          } else if (mx > m_used + kRescaleThreshold) {
            alpha = ex2(m_used - mx);                  // 0 when nothing was accumulated yet
            m_used = mx;
          }
          if (j > lo && __any_sync(0xffffffffu, alpha != 1.f)) {
            // S(j) is complete, so every earlier P V product has finished; the next one waits for p_ready below:
            // nobody else touches O now
#pragma unroll
            for (int c = 0; c < HV / 16; ++c) {
              uint32_t r[16];
              tmem_ld_32x32b_x16(o_tmem + c * 16, r);
              tmem_ld_wait();
#pragma unroll
              for (int i = 0; i < 16; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * alpha);
              tmem_st_32x32b_x16(o_tmem + c * 16, r);
            }
          }
          const float neg_m = (m_used == -INFINITY) ? 0.f : -m_used;
          const uint64_t negm2 = pack2(neg_m, neg_m);
          uint64_t rs2[4] = {0, 0, 0, 0};
          // exp2 of the scaled, shifted scores two at a time; P goes back as bf16 pairs, 64 score columns (32 packed
          // registers) per store, into the first 64 columns of this tile's S buffer
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            // pass 2: 64 scores at a time; the second half is read before the first half's P overwrites columns 0..31
            if (MASK && (hi_max < h * 64 || lo_min > h * 64 + 63)) {
              uint32_t zero[32];
#pragma unroll
              for (int i = 0; i < 32; ++i) zero[i] = 0u;
              tmem_st_32x32b_x32(s_tmem + h * 32, zero);
              continue;
            }
            uint32_t sr[64];
            {
              uint32_t (&ra)[32] = *reinterpret_cast<uint32_t(*)[32]>(&sr[0]);
              uint32_t (&rb)[32] = *reinterpret_cast<uint32_t(*)[32]>(&sr[32]);
              tmem_ld_32x32b_x32(s_tmem + h * 64, ra);
              tmem_ld_32x32b_x32(s_tmem + h * 64 + 32, rb);
              tmem_ld_wait();
            }
            float* s = reinterpret_cast<float*>(sr);
            if constexpr (CAP) {
              // capped, shifted scores: by the polynomial where every score of the warp is within its reach
              float am = 0.f;
#pragma unroll
              for (int i = 0; i < 32; ++i) am = fmax3(am, fabsf(s[2 * i]), fabsf(s[2 * i + 1]));
              if (__all_sync(0xffffffffu, am * args.cap_scale <= kPolyReach)) {
                uint64_t c[5];
#pragma unroll
                for (int k = 0; k < 5; ++k) c[k] = pack2(args.cap_poly[k], args.cap_poly[k]);
#pragma unroll
                for (int i = 0; i < 32; ++i) {
                  const uint64_t v = pack2(s[2 * i], s[2 * i + 1]);
                  const uint64_t z = mul2(v, v);
                  unpack2(fma2(v, fma2(fma2(fma2(fma2(c[4], z, c[3]), z, c[2]), z, c[1]), z, c[0]), negm2), s[2 * i], s[2 * i + 1]);
                }
              } else {
#pragma unroll
                for (int i = 0; i < 64; ++i) s[i] = capped(s[i] * args.cap_scale, args.cap_log2) + neg_m;
              }
            }
#pragma unroll
            for (int a = 0; a < 2; ++a) {
              if (MASK && hi_min < h * 64 + a * 32 + 31) {
#pragma unroll
                for (int i = a * 32; i < a * 32 + 32; ++i)
                  if (h * 64 + i > col_hi) s[i] = -INFINITY;
              }
              if (MASK && lo_max > h * 64 + a * 32) {
#pragma unroll
                for (int i = a * 32; i < a * 32 + 32; ++i)
                  if (h * 64 + i < col_lo) s[i] = -INFINITY;
              }
            }
            uint32_t pk[32];
#pragma unroll
            for (int i = 0; i < 32; ++i) {
              float t0, t1;
              if constexpr (CAP) { t0 = s[2 * i]; t1 = s[2 * i + 1]; }
              else unpack2(fma2(pack2(s[2 * i], s[2 * i + 1]), scale2, negm2), t0, t1);
              const float e0 = ex2(t0), e1 = ex2(t1);
              rs2[i & 3] = add2(rs2[i & 3], pack2(e0, e1));
              pk[i] = pack_bf16x2(e0, e1);
            }
            tmem_st_32x32b_x32(s_tmem + h * 32, pk);
          }
          float r0, r1, r2, r3;
          unpack2(add2(rs2[0], rs2[1]), r0, r1);
          unpack2(add2(rs2[2], rs2[3]), r2, r3);
          l_sum = l_sum * alpha + ((r0 + r1) + (r2 + r3));
        };
        if (lo_max > 0 || hi_min < kTile - 1) softmax_tile(std::true_type{});
        else softmax_tile(std::false_type{});
        tmem_st_wait();
        tc_fence_before();
        mbar_arrive(smem_u32(p_ready));
      }
      if (ok) ok = mbar_wait(smem_u32(pv_done), (it - 1) & 1, abort_flag, args.status, kStatusWaitTimeoutEpilogue);
      // one decision for the whole warpgroup (a thread that gave up above still arrives here)
      ok = named_bar_and(2, 128, ok);
      if (!ok) break;
      tc_fence_after();
      // the sink joins the denominator on the scale of the sum; an enormous sink overflows to a zero weight of the keys
      const float den = args.sink ? l_sum + ex2(args.sink[t.head] * 1.4426950408889634f - m_used) : l_sum;
      const float inv_l = args.out_scale / den;
      // 32 columns at a time through 2 KB of shared memory per warp, so that a store covers 64 bytes of eight rows each
      uint8_t* stage = sOut + ew * 2048;
      __nv_bfloat16* obase = args.out + (t.q0 + ew * 32) * args.ld_out + static_cast<size_t>(t.head * args.vheads + t.vsel) * args.DV;
#pragma unroll
      for (int c = 0; c < HV / 32; ++c) {
        uint32_t r[32];
        tmem_ld_32x32b_x32(o_tmem + c * 32, r);
        tmem_ld_wait();
#pragma unroll
        for (int q = 0; q < 4; ++q)
          *reinterpret_cast<uint4*>(stage + lane * 64 + ((q ^ ((lane >> 1) & 3)) << 4)) = make_uint4(
              pack_bf16x2(__uint_as_float(r[q * 8 + 0]) * inv_l, __uint_as_float(r[q * 8 + 1]) * inv_l),
              pack_bf16x2(__uint_as_float(r[q * 8 + 2]) * inv_l, __uint_as_float(r[q * 8 + 3]) * inv_l),
              pack_bf16x2(__uint_as_float(r[q * 8 + 4]) * inv_l, __uint_as_float(r[q * 8 + 5]) * inv_l),
              pack_bf16x2(__uint_as_float(r[q * 8 + 6]) * inv_l, __uint_as_float(r[q * 8 + 7]) * inv_l));
        __syncwarp();
        const int col = c * 32 + (lane & 3) * 8;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int rr = i * 8 + (lane >> 2);
          if (ew * 32 + rr < t.rows && col < args.DV)
            *reinterpret_cast<uint4*>(obase + rr * args.ld_out + col) =
                *reinterpret_cast<const uint4*>(stage + rr * 64 + (((lane & 3) ^ ((rr >> 1) & 3)) << 4));
        }
        __syncwarp();
      }
      // O is read: the next tile's first P V product, which overwrites it, waits for this warpgroup's next p_ready
      tc_fence_before();
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 256);
  }
}

// ---- every head's weights on the values of every key / value head ---------------------------------------------------------------
// The products with the values are G times those of ordinary attention, so scores and softmax of a key tile serve NV = 256 / HV
// value heads at once: their accumulators fill half of tensor memory, two score buffers the other half, and one CTA owns the SM.
// The scores of key tile j + 1 are computed before the products of tile j with the values, under which their softmax then runs.
// Eight softmax warps share a query tile: a row belongs to two threads, 64 key columns each, which exchange their maxima (and, at
// the end, their sums) through shared memory and keep the scores in registers in between; each writes one half of the results.
//
// Roles (320 threads): warp 0 TMA producer, warp 1 MMA issuer + TMEM owner, warps 2..9 softmax. Every wait is bounded.
constexpr int kAvThreads = 320;
constexpr int kAvRing = 96 * 1024;         // V tiles

template <int HQ, int HV>
__global__ void __launch_bounds__(kAvThreads, 1)
paged_prefill_values_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                            const __grid_constant__ CUtensorMap tmV, const Args args, const int G) {
  constexpr int QB = HQ / 64, VB = HV / 64, NV = 256 / HV;
  constexpr int kQBytes = QB * kSubBytes, kVBytes = VB * kSubBytes, kSlots = kAvRing / kVBytes;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + kQBytes;                        // two stages
  uint8_t* sV = sK + 2 * kQBytes;                    // ring
  uint8_t* sOut = sV + kAvRing;                      // 2 KB per softmax warp
  float* sMax = reinterpret_cast<float*>(sOut + 8 * 2048);        // [2 tiles][2 halves][128]
  float* sSum = sMax + 4 * kTile;                    // [2 halves][128]
  uint64_t* bars = reinterpret_cast<uint64_t*>(sSum + 2 * kTile);
  uint64_t* q_full = bars;
  uint64_t* q_empty = bars + 1;
  uint64_t* k_full = bars + 2;                       // 2
  uint64_t* k_empty = bars + 4;                      // 2
  uint64_t* s_full = bars + 6;                       // 2
  uint64_t* p_ready = bars + 8;
  uint64_t* pv_done = bars + 9;                      // 2: a tile's softmax may end before the products of the tile before
  uint64_t* v_full = bars + 11;                      // kSlots
  uint64_t* v_empty = v_full + kSlots;
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(v_empty + kSlots);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_holder + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int vblocks = (G + NV - 1) / NV;
  struct Tile { int b, head, v0, nv, q0, rows, pos0, lo, n_kv; };     // value heads v0 .. v0 + nv - 1, key tiles lo .. n_kv - 1
  auto first_of = [&](int pos) {
    int lo = args.chunk > 0 ? pos - pos % args.chunk : 0;
    if (args.window > 0 && pos - args.window + 1 > lo) lo = pos - args.window + 1;
    return lo;
  };
  auto tile_of = [&](int item) {
    Tile t;
    t.v0 = item % vblocks * NV;
    t.nv = G - t.v0 < NV ? G - t.v0 : NV;
    item /= vblocks;
    const int4 w = args.work[item / args.num_q_heads];
    t.head = item % args.num_q_heads;
    t.b = w.x; t.q0 = w.y; t.rows = w.z; t.pos0 = w.w;
    t.lo = first_of(t.pos0) / kTile;
    t.n_kv = (t.pos0 + t.rows - 1) / kTile + 1;
    return t;
  };
  const int first_item = static_cast<int>(blockIdx.x), step = static_cast<int>(gridDim.x);

  if (threadIdx.x == 0) {
    *abort_flag = 0;
    for (int i = 0; i < 11 + 2 * kSlots; ++i) mbar_init(smem_u32(&bars[i]), &bars[i] == p_ready ? 256 : 1);
    fence_barrier_init();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_holder), 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_holder;
  const uint32_t tmem_O = tmem_base + 2 * kTile;     // P of a tile lives in the first 64 columns of its scores

  if (warp == 0) {
    // ------------------------------ TMA producer (the whole warp, one lane issues) ------------------------------
    const bool leader = elect_one();
    const int bs = args.block_size;
    uint32_t it = 0, n = 0, unit = 0;                // key tiles, query tiles and V tiles so far
    bool ok = true;
    // wait until a buffer is free (the lanes agree on the outcome) and announce what goes there
    auto claim = [&](uint64_t* empty, uint32_t parity, uint64_t* full, uint32_t bytes) {
      ok = mbar_wait(smem_u32(empty), parity, abort_flag, args.status, kStatusWaitTimeoutProducer);
      ok = __all_sync(0xffffffffu, ok);
      if (ok && leader) mbar_expect_tx(smem_u32(full), bytes);
      __syncwarp();
    };
    for (int item = first_item; item < args.n_items && ok; item += step, ++n) {
      const Tile t = tile_of(item);
      const int* table = args.block_tables + static_cast<size_t>(t.b) * args.max_blocks;
      const int end = t.pos0 + t.rows, kcol = t.head / args.group * args.D;
      int page = tile_page(table, bs, t.lo * kTile, end);
      claim(q_empty, (n & 1) ^ 1, q_full, kQBytes);
      if (!ok) break;
      if (leader)
        for (int c = 0; c < QB; ++c) tma_load_3d(smem_u32(sQ) + c * kSubBytes, &tmQ, smem_u32(q_full), c * 64, t.head, t.q0);
      __syncwarp();
      auto load_k = [&](int pg) {
        const int st = it & 1;
        claim(&k_empty[st], ((it >> 1) & 1) ^ 1, &k_full[st], kQBytes);
        if (!ok) return;
        tma_load_pages(leader, smem_u32(sK) + st * kQBytes, kSubBytes, &tmK, smem_u32(&k_full[st]), pg, bs, kcol, QB);
        ++it;
      };
      load_k(page);
      for (int j = t.lo; j < t.n_kv && ok; ++j) {
        const int next = j + 1 < t.n_kv ? tile_page(table, bs, (j + 1) * kTile, end) : 0;
        if (j + 1 < t.n_kv) load_k(next);
        for (int v = 0; v < t.nv && ok; ++v, ++unit) {
          const int slot = unit % kSlots;
          claim(&v_empty[slot], ((unit / kSlots) & 1) ^ 1, &v_full[slot], kVBytes);
          if (ok)
            tma_load_pages(leader, smem_u32(sV) + slot * kVBytes, kSubBytes, &tmV, smem_u32(&v_full[slot]), page, bs,
                           (t.v0 + v) * args.DV, VB);
        }
        page = next;
      }
    }
  } else if (warp == 1) {
    // ------------------------------ MMA issuer (the whole warp, one lane issues) ------------------------------
    constexpr uint32_t IDESC_QK = umma_idesc_bf16(kTile, kTile, 0, 0);
    constexpr uint32_t IDESC_PV = umma_idesc_bf16(kTile, HV, 0, 1);
    const bool leader = elect_one();
    const uint64_t q_desc = umma_desc_kmajor_sw128(smem_u32(sQ));
    uint32_t it = 0, n = 0, unit = 0;
    bool ok = true, first_key = true;                // first_key: the pending products start their query tile's sums
    int pending = 0;                                 // value heads of the pending products
    auto wait = [&](uint64_t* bar, uint32_t parity) {
      ok = mbar_wait(smem_u32(bar), parity, abort_flag, args.status, kStatusWaitTimeoutMma);
      ok = __all_sync(0xffffffffu, ok);
    };
    // O(v) (+)= P V(v) of key tile it - 1
    auto issue_pv = [&]() {
      wait(p_ready, (it - 1) & 1);
      const uint32_t pa = tmem_base + ((it - 1) & 1) * kTile;
      for (int v = 0; v < pending && ok; ++v, ++unit) {
        const int slot = unit % kSlots;
        wait(&v_full[slot], (unit / kSlots) & 1);
        if (!ok) return;
        tc_fence_after();
        const uint64_t v_desc = umma_desc_mnmajor_sw128(smem_u32(sV) + slot * kVBytes, kSubBytes);
        const uint32_t o = tmem_O + v * HV;
#pragma unroll
        for (int k = 0; k < kTile / 16; ++k)
          umma_f16_ts_warp(leader, o, pa + k * 8, v_desc + ((k * 16 * 128) >> 4), IDESC_PV, (!first_key || k > 0) ? 1u : 0u);
        umma_commit_warp(leader, smem_u32(&v_empty[slot]));
      }
      if (ok) umma_commit_warp(leader, smem_u32(&pv_done[(it - 1) & 1]));
    };
    for (int item = first_item; item < args.n_items && ok; item += step, ++n) {
      const Tile t = tile_of(item);
      for (int j = t.lo; j < t.n_kv && ok; ++j) {
        if (j == t.lo) {
          if (it > 0) issue_pv();                    // the last products of the query tile before do not wait for this one's q
          if (ok) wait(q_full, n & 1);
        }
        const int st = it & 1;
        if (ok) wait(&k_full[st], (it >> 1) & 1);
        if (!ok) break;
        tc_fence_after();
        // these scores overwrite those whose products with the values were issued before the last ones
        const uint64_t k_desc = umma_desc_kmajor_sw128(smem_u32(sK) + st * kQBytes);
        const uint32_t s_tmem = tmem_base + st * kTile;
#pragma unroll
        for (int k = 0; k < HQ / 16; ++k) {
          constexpr int kSubUnits = kSubBytes >> 4;
          const int off = (k >> 2) * kSubUnits + (k & 3) * 2;
          umma_f16_ss_warp(leader, s_tmem, q_desc + off, k_desc + off, IDESC_QK, k > 0 ? 1u : 0u);
        }
        umma_commit_warp(leader, smem_u32(&s_full[st]));
        umma_commit_warp(leader, smem_u32(&k_empty[st]));
        if (j == t.n_kv - 1) umma_commit_warp(leader, smem_u32(q_empty));
        if (j > t.lo) issue_pv();
        first_key = j == t.lo;
        pending = t.nv;
        ++it;
      }
    }
    if (ok && it > 0) issue_pv();
  } else {
    // ------------------------------ softmax warpgroups ------------------------------
    const int ew = warp & 3, half = (warp - 2) >> 2;
    const int row = ew * 32 + lane;
    const uint32_t lane_base = static_cast<uint32_t>(ew * 32) << 16;
    bool ok = true;
    const uint64_t scale2 = pack2(args.scale_log2, args.scale_log2);
    uint32_t it = 0;
    for (int item = first_item; item < args.n_items; item += step) {
      const Tile t = tile_of(item);
      const int my_pos = t.pos0 + row, my_first = first_of(my_pos);
      float m_used = -INFINITY, l_sum = 0.f;
      for (int j = t.lo; j < t.n_kv; ++j, ++it) {
        const uint32_t s_tmem = tmem_base + (it & 1) * kTile + lane_base;
        ok = mbar_wait(smem_u32(&s_full[it & 1]), (it >> 1) & 1, abort_flag, args.status, kStatusWaitTimeoutEpilogue) && ok;
        tc_fence_after();
        uint32_t sr[64];
        {
          uint32_t (&ra)[32] = *reinterpret_cast<uint32_t(*)[32]>(&sr[0]);
          uint32_t (&rb)[32] = *reinterpret_cast<uint32_t(*)[32]>(&sr[32]);
          tmem_ld_32x32b_x32(s_tmem + half * 64, ra);
          tmem_ld_32x32b_x32(s_tmem + half * 64 + 32, rb);
          tmem_ld_wait();
        }
        float* s = reinterpret_cast<float*>(sr);
        // columns [col_lo, col_hi] of this half are visible to the row; the bounds grow with the row
        const int col_lo = my_first - j * kTile - half * 64, col_hi = my_pos - j * kTile - half * 64;
        if (__shfl_sync(0xffffffffu, col_hi, 0) < 63 || __shfl_sync(0xffffffffu, col_lo, 31) > 0) {
#pragma unroll
          for (int i = 0; i < 64; ++i)
            if (i > col_hi || i < col_lo) s[i] = -INFINITY;
        }
        float mxs[4];
#pragma unroll
        for (int a = 0; a < 4; ++a) {
          float m = s[a * 16];
#pragma unroll
          for (int i = 1; i + 1 < 16; i += 2) m = fmax3(m, s[a * 16 + i], s[a * 16 + i + 1]);
          mxs[a] = fmaxf(m, s[a * 16 + 15]);
        }
        float* mx_of = sMax + (it & 1) * 2 * kTile;
        mx_of[half * kTile + row] = fmaxf(fmaxf(mxs[0], mxs[1]), fmaxf(mxs[2], mxs[3])) * args.scale_log2;
        named_bar_sync(1, 256);                      // both halves have their scores in registers, too
        const float mx = fmaxf(mx_of[row], mx_of[kTile + row]);
        float alpha = 1.f;
        if (j == t.lo) {
          m_used = mx;
        } else if (mx > m_used + kRescaleThreshold) {
          alpha = ex2(m_used - mx);
          m_used = mx;
        }
        if (j > t.lo && __any_sync(0xffffffffu, alpha != 1.f)) {
          // products up to tile j - 1 have to be complete; the next ones wait for p_ready below
          ok = mbar_wait(smem_u32(&pv_done[(it - 1) & 1]), ((it - 1) >> 1) & 1, abort_flag, args.status, kStatusWaitTimeoutEpilogue) && ok;
          tc_fence_after();
#pragma unroll 1
          for (int c = 0; c < 8; ++c) {
            uint32_t r[16];
            const uint32_t o = tmem_O + lane_base + half * 128 + c * 16;
            tmem_ld_32x32b_x16(o, r);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 16; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * alpha);
            tmem_st_32x32b_x16(o, r);
          }
        }
        const float neg_m = m_used == -INFINITY ? 0.f : -m_used;
        const uint64_t negm2 = pack2(neg_m, neg_m);
        uint64_t rs2[4] = {0, 0, 0, 0};
        uint32_t pk[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          float x0, x1;
          unpack2(fma2(pack2(s[2 * i], s[2 * i + 1]), scale2, negm2), x0, x1);
          const float e0 = ex2(x0), e1 = ex2(x1);
          rs2[i & 3] = add2(rs2[i & 3], pack2(e0, e1));
          pk[i] = pack_bf16x2(e0, e1);
        }
        tmem_st_32x32b_x32(s_tmem + half * 32, pk);
        float r0, r1, r2, r3;
        unpack2(add2(rs2[0], rs2[1]), r0, r1);
        unpack2(add2(rs2[2], rs2[3]), r2, r3);
        l_sum = l_sum * alpha + ((r0 + r1) + (r2 + r3));
        tmem_st_wait();
        tc_fence_before();
        mbar_arrive(smem_u32(p_ready));
      }
      ok = mbar_wait(smem_u32(&pv_done[(it - 1) & 1]), ((it - 1) >> 1) & 1, abort_flag, args.status, kStatusWaitTimeoutEpilogue) && ok;
      sSum[half * kTile + row] = l_sum;
      ok = named_bar_and(2, 256, ok);
      if (!ok) break;
      tc_fence_after();
      const float inv_l = args.out_scale / (sSum[row] + sSum[kTile + row]);
      uint8_t* stage = sOut + (half * 4 + ew) * 2048;
      __nv_bfloat16* obase = args.out + (t.q0 + ew * 32) * args.ld_out + static_cast<size_t>(t.head * G + t.v0) * args.DV;
#pragma unroll 1
      for (int c = 0; c < 4; ++c) {
        const int at = half * 128 + c * 32, v = at / HV, col0 = at % HV;
        uint32_t r[32];
        tmem_ld_32x32b_x32(tmem_O + lane_base + at, r);
        tmem_ld_wait();
#pragma unroll
        for (int q = 0; q < 4; ++q)
          *reinterpret_cast<uint4*>(stage + lane * 64 + ((q ^ ((lane >> 1) & 3)) << 4)) = make_uint4(
              pack_bf16x2(__uint_as_float(r[q * 8 + 0]) * inv_l, __uint_as_float(r[q * 8 + 1]) * inv_l),
              pack_bf16x2(__uint_as_float(r[q * 8 + 2]) * inv_l, __uint_as_float(r[q * 8 + 3]) * inv_l),
              pack_bf16x2(__uint_as_float(r[q * 8 + 4]) * inv_l, __uint_as_float(r[q * 8 + 5]) * inv_l),
              pack_bf16x2(__uint_as_float(r[q * 8 + 6]) * inv_l, __uint_as_float(r[q * 8 + 7]) * inv_l));
        __syncwarp();
        const int col = col0 + (lane & 3) * 8;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int rr = i * 8 + (lane >> 2);
          if (ew * 32 + rr < t.rows && col < args.DV && v < t.nv)
            *reinterpret_cast<uint4*>(obase + rr * args.ld_out + v * args.DV + col) =
                *reinterpret_cast<const uint4*>(stage + rr * 64 + (((lane & 3) ^ ((rr >> 1) & 3)) << 4));
        }
        __syncwarp();
      }
      // O is read: the next query tile's first products, which overwrite it, wait for the warps' next p_ready
      tc_fence_before();
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

template <int HQ, int HV>
int launch_values(const CUtensorMap& tQ, const CUtensorMap& tK, const CUtensorMap& tV, Args a, int n_work, int G, cudaStream_t stream) {
  constexpr int NV = 256 / HV, SLOTS = kAvRing / (HV / 64 * kSubBytes);
  constexpr int SMEM = 3 * (HQ / 64 * kSubBytes) + kAvRing + 8 * 2048 + 6 * kTile * 4 + (11 + 2 * SLOTS) * 8 + 16 + 1024;
  static_assert(SMEM <= 232448, "shared memory budget exceeded");
  auto kern = paged_prefill_values_kernel<HQ, HV>;
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM) != cudaSuccess) {
      mfb_host::set_error("paged_prefill_tc: cannot raise the shared memory limit");
      return 10;
    }
    attr_set = true;
  }
  a.n_items = n_work * a.num_q_heads * ((G + NV - 1) / NV);
  kern<<<a.n_items < 148 ? a.n_items : 148, kAvThreads, SMEM, stream>>>(tQ, tK, tV, a, G);
  if (cudaGetLastError() != cudaSuccess) { mfb_host::set_error("paged_prefill_tc: launch failed"); return 11; }
  return 0;
}

// three-dimensional map of q [T, Hq, D]: box of 128 tokens x 1 head x 64 columns; columns past D read as zero
int make_q_map(CUtensorMap* out, const void* q, uint64_t T, uint64_t Hq, uint64_t D) {
  mfb_host::EncodeTiledFn enc = mfb_host::get_encode_tiled();
  if (!enc) { mfb_host::set_error("cuTensorMapEncodeTiled entry point not available"); return 1; }
  if ((reinterpret_cast<uintptr_t>(q) & 15) || (D * 2) % 16) { mfb_host::set_error("paged_prefill_tc: q not aligned"); return 2; }
  cuuint64_t gdim[3] = {D, Hq, T};
  cuuint64_t gstride[2] = {D * 2, Hq * D * 2};
  cuuint32_t box[3] = {64, 1, kTile};
  cuuint32_t estr[3] = {1, 1, 1};
  const CUresult r = enc(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(q), gdim, gstride, box, estr,
                         CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                         CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) { mfb_host::set_error("paged_prefill_tc: tensor map of q failed (%d)", (int)r); return 3; }
  return 0;
}

template <int HQ, int HV, bool CAP>
int launch(const CUtensorMap& tQ, const CUtensorMap& tK, const CUtensorMap& tV, const Args& a, int max_ctas, cudaStream_t stream) {
  constexpr int QBYTES = HQ / 64 * kSubBytes, VBYTES = HV / 64 * kSubBytes;
  constexpr int SMEM = 2 * QBYTES + VBYTES + 4 * 2048 + 9 * 8 + 16 + 1024;
  static_assert((HQ > 128 ? 1 : 2) * SMEM <= 232448, "shared memory budget exceeded");
  auto kern = paged_prefill_tc_kernel<HQ, HV, CAP>;
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM) != cudaSuccess) {
      mfb_host::set_error("paged_prefill_tc: cannot raise the shared memory limit");
      return 10;
    }
    attr_set = true;
  }
  const int grid = a.n_items < max_ctas ? a.n_items : max_ctas;
  kern<<<grid, kThreads, SMEM, stream>>>(tQ, tK, tV, a);
  if (cudaGetLastError() != cudaSuccess) { mfb_host::set_error("paged_prefill_tc: launch failed"); return 11; }
  return 0;
}

}  // namespace ppt
}  // namespace mfb

extern "C" {
using namespace mfb;

// 1 when the kernel serves these shapes (bf16): sizes are multiples of 8 up to 128, the block size divides 128.
int mfb_paged_prefill_tc_supported(int Hq, int Hkv, int D, int DV, int block_size) {
  if (Hkv < 1 || Hq < 1 || Hq % Hkv || D < 8 || DV < 8 || D > 128 || DV > 128 || D % 8 || DV % 8) return 0;
  return (block_size == 16 || block_size == 32 || block_size == 64 || block_size == 128) ? 1 : 0;
}

// The same for keys of up to 192 numbers, without all_values or a soft cap beyond 128.
int mfb_paged_prefill_tc_wide_supported(int Hq, int Hkv, int D, int DV, int block_size) {
  return D <= 192 && D % 8 == 0 ? mfb_paged_prefill_tc_supported(Hq, Hkv, D < 128 ? D : 128, DV, block_size) : 0;
}

// q [T, Hq, D], caches [num_blocks, block_size, Hkv, D | DV] with rows ld_k / ld_v elements apart, out [T, Hq, DV] (all_values:
// [T, Hq, Hkv, DV]), all bf16. chunk > 0: a position sees its own chunk only; window > 0: itself and the window - 1 positions
// before it. work [n_work, 4] int32: (sequence,
// first row of q, 1..128 rows, position of the first row) per query tile, heaviest first; the rows' keys are in the cache.
// persistent: two CTAs per SM walk over all tiles (for tiles of a few key tiles); else a CTA per query tile and head, which
// balances tiles of very different lengths better. softcap > 0: scores become softcap * tanh(score / softcap). Rows of out lie
// ld_out elements apart; the result is multiplied by out_scale.
int mfb_paged_prefill_tc(const void* q, const void* key_cache, const void* value_cache, const int* work, int n_work, int persistent,
                         const int* block_tables, const float* sink, void* out, int T,
                         int Hq, int Hkv, int D, int DV, int num_blocks, int block_size, int max_blocks, int chunk, int window,
                         int all_values, long long ld_k, long long ld_v, float scale, float softcap, long long ld_out,
                         float out_scale, int* status, cudaStream_t stream) {
  if (!mfb_paged_prefill_tc_wide_supported(Hq, Hkv, D, DV, block_size) || (D > 128 && (all_values || softcap > 0.f)) ||
      num_blocks < 1 || T < 1) {
    mfb_host::set_error("paged_prefill_tc: unsupported Hq=%d Hkv=%d D=%d DV=%d block_size=%d", Hq, Hkv, D, DV, block_size);
    return 1;
  }
  if (n_work <= 0) return 0;
  if (ld_k < (long long)Hkv * D || ld_v < (long long)Hkv * DV) {
    mfb_host::set_error("paged_prefill_tc: row pitches %lld and %lld", ld_k, ld_v);
    return 1;
  }
  if (ld_out % 8 || (reinterpret_cast<uintptr_t>(out) & 15)) {
    mfb_host::set_error("paged_prefill_tc: rows of the result must start on 16 bytes");
    return 1;
  }
  CUtensorMap tQ, tK, tV;
  int rc;
  const CUtensorMapDataType BF = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  const uint64_t rows = (uint64_t)num_blocks * block_size;
  if ((rc = mfb_host::make_tmap_2d(&tK, key_cache, 2, BF, rows, (uint64_t)Hkv * D, (uint64_t)ld_k, block_size, 64))) return 30 + rc;
  if ((rc = mfb_host::make_tmap_2d(&tV, value_cache, 2, BF, rows, (uint64_t)Hkv * DV, (uint64_t)ld_v, block_size, 64))) return 40 + rc;
  if ((rc = ppt::make_q_map(&tQ, q, T, Hq, D))) return 20 + rc;
  ppt::Args a;
  a.work = reinterpret_cast<const int4*>(work); a.vheads = all_values ? Hkv : 1; a.n_items = n_work * Hq * a.vheads;
  a.block_tables = block_tables; a.sink = sink;
  a.out = reinterpret_cast<__nv_bfloat16*>(out);
  a.num_q_heads = Hq; a.group = Hq / Hkv; a.D = D; a.DV = DV; a.block_size = block_size; a.max_blocks = max_blocks;
  a.chunk = chunk; a.window = window; a.scale_log2 = scale * 1.4426950408889634f; a.status = status;
  a.cap_log2 = softcap > 0.f ? softcap * 1.4426950408889634f : 0.f;
  a.cap_scale = softcap > 0.f ? scale / softcap : 0.f;
  float power = a.scale_log2;
  for (int k = 0; k < 5; ++k, power *= a.cap_scale * a.cap_scale) a.cap_poly[k] = ppt::kTanhRatio[k] * power;
  a.ld_out = ld_out; a.out_scale = out_scale;
  if (a.vheads > 1 && !sink && !(softcap > 0.f)) {
    if (D > 64) return DV > 64 ? ppt::launch_values<128, 128>(tQ, tK, tV, a, n_work, Hkv, stream)
                               : ppt::launch_values<128, 64>(tQ, tK, tV, a, n_work, Hkv, stream);
    return DV > 64 ? ppt::launch_values<64, 128>(tQ, tK, tV, a, n_work, Hkv, stream)
                   : ppt::launch_values<64, 64>(tQ, tK, tV, a, n_work, Hkv, stream);
  }
  const int max_ctas = persistent ? (D > 128 ? 1 : 2) * 148 : a.n_items;
#define MFB_PPT(HQ_, HV_) \
  return softcap > 0.f ? ppt::launch<HQ_, HV_, true>(tQ, tK, tV, a, max_ctas, stream) : ppt::launch<HQ_, HV_, false>(tQ, tK, tV, a, max_ctas, stream)
  if (D > 128)
    return DV > 64 ? ppt::launch<192, 128, false>(tQ, tK, tV, a, max_ctas, stream)
                   : ppt::launch<192, 64, false>(tQ, tK, tV, a, max_ctas, stream);
  if (D > 64) {
    if (DV > 64) MFB_PPT(128, 128);
    MFB_PPT(128, 64);
  }
  if (DV > 64) MFB_PPT(64, 128);
  MFB_PPT(64, 64);
#undef MFB_PPT
}

}  // extern "C"
