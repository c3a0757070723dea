// Decode attention whose softmax weights are mixed over heads, over a paged bf16 cache (sm_100a, tcgen05 + TMA):
//     w_g[t] = softmax over the visible t of scale <q_g, k_own(g)[t]>          g = 0 .. H - 1, own(g) = g / (H / G)
//     out_h  = sigmoid(gate_h) * sum_g talk[h, g] * sum_t w_g[t] v_own(h)[t]
// Every head's weights meet the values of every key / value head, so a CTA takes (split of the sequence, sequence) with ALL query
// heads: it reads each key and each value once, where one CTA per key / value head would read the values G times.
//
// As in paged_decode_tc.cu the products are transposed, so that 128 tokens fill the rows of the tensor core:
//     S^T(i) [128 tokens x 16]  = K_own . Q_i^T             i: up to 16 heads of one key / value head; a buffer of its own each
//     O^T(v) [128 x Hp heads]  += V_v^T . P^T               v: every value head; Hp: the heads, padded to a multiple of 16
// K and V tiles stream through a ring in the order K(0, *), then K(j + 1, *), V(j, *), so the scores of the next tile are
// computed under the softmax of this one. Scores and weights of two tiles are in flight. The running maximum of a head is kept in
// shared memory, its sum per token row. Where the accumulators of all value heads do not fit tensor memory, blockIdx.y takes a
// part of them. The splits are merged, mixed and gated by talk_combine_kernel.
//
// Roles (192 threads): warp 0 TMA producer, warp 1 MMA issuer + TMEM owner, warps 2..5 softmax / epilogue. Every wait is bounded.
#include "common.cuh"

namespace mfb {
namespace ptd {

constexpr int kThreads = 192;
constexpr int kTile = 128;
constexpr int kItem = 16;                  // score columns of an item
constexpr int kSub = kTile * 128;          // [128 tokens][64 columns] swizzled sub-tile, 16 KB
constexpr int kUnit = 2 * kSub;
constexpr int kQItem = 2 * kItem * 128;    // two [16 heads][64 columns] sub-tiles
constexpr int kMaxItems = 16, kMaxHeads = 64, kMaxSlots = 6;
constexpr float kRescale = 8.0f;
constexpr int kSmemLimit = 232448;

struct Args {
  const int* block_tables;   // [B, max_blocks]
  const int* context_lens;   // [B]
  const int* cu_q;           // [B + 1] or null: only sequences with exactly one new row are computed
  int max_blocks, block_size, H, G, group, splits, D, DV, window;
  int per_kv, items, Hp, nv, slots, tmem_cols;    // items per KV head, items, padded heads, value heads per CTA, ring slots
  float scale_log2;
  float* part_acc;           // [B, H, G, splits, DV] unnormalised
  float* part_ml;            // [B, H, splits, 2]: running max (log2 units), sum
  int* status;
};

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm volatile("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__host__ __device__ constexpr int fixed_bytes(int Hp, int items) {
  return 2 * 2 * Hp * 128 + items * kQItem + Hp * kTile * 4 + 6 * kMaxHeads * 4 +
         (8 + 2 * kMaxSlots + 2 * kMaxItems) * 8 + 16 + 1024;
}

__global__ void __launch_bounds__(kThreads, 1)
paged_talk_decode_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                         const __grid_constant__ CUtensorMap tmV, const Args args) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const int Hp = args.Hp, items = args.items, slots = args.slots, nv_max = args.nv;
  const int p_sub = Hp * 128, p_buf = 2 * p_sub;
  uint8_t* sRing = smem;
  uint8_t* sP = sRing + slots * kUnit;                      // two buffers of two [Hp heads][64 tokens] sub-tiles
  uint8_t* sQ = sP + 2 * p_buf;
  float* sL = reinterpret_cast<float*>(sQ + items * kQItem);          // [Hp][128] sums per token row
  float* sM = sL + Hp * kTile;                              // [kMaxHeads] running maxima
  float* sAlpha = sM + kMaxHeads;                           // [kMaxHeads]
  float* red = sAlpha + kMaxHeads;                          // [4 warps][kMaxHeads]
  uint64_t* bars = reinterpret_cast<uint64_t*>(red + 4 * kMaxHeads);
  uint64_t* q_full = bars;
  uint64_t* p_ready = bars + 1;
  uint64_t* pv_done = bars + 2;
  uint64_t* s_empty = bars + 3;                             // 2
  uint64_t* full = bars + 5;                                // slots
  uint64_t* empty = full + kMaxSlots;
  uint64_t* s_full = empty + kMaxSlots;                     // [2][items]
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(s_full + 2 * kMaxItems);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_holder + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int split = blockIdx.x, v0 = blockIdx.y * nv_max, b = blockIdx.z;
  const int nv = min(nv_max, args.G - v0);
  int q_row = b;
  if (args.cu_q) {
    q_row = args.cu_q[b];
    if (args.cu_q[b + 1] - q_row != 1) return;
  }
  const int len = args.context_lens[b];
  const int first_tok = args.window > 0 && len > args.window ? len - args.window : 0;
  const int base_tile = first_tok / kTile;
  const int n_tiles_all = (len + kTile - 1) / kTile - base_tile;
  const int per = (n_tiles_all + args.splits - 1) / args.splits;
  const int rel0 = split * per;
  const int rel1 = rel0 + per < n_tiles_all ? rel0 + per : n_tiles_all;
  const int n_tiles = rel1 > rel0 ? rel1 - rel0 : 0;
  const int t0 = base_tile + rel0;
  const int k_halves = args.D > 64 ? 2 : 1, v_halves = args.DV > 64 ? 2 : 1;

  if (threadIdx.x == 0) {
    *abort_flag = 0;
    mbar_init(smem_u32(q_full), 1);
    mbar_init(smem_u32(p_ready), 128);
    mbar_init(smem_u32(pv_done), 1);
    for (int s = 0; s < 2; ++s) mbar_init(smem_u32(&s_empty[s]), 128);
    for (int s = 0; s < slots; ++s) {
      mbar_init(smem_u32(&full[s]), 1);
      mbar_init(smem_u32(&empty[s]), 1);
    }
    for (int s = 0; s < 2 * items; ++s) mbar_init(smem_u32(&s_full[s]), 1);
    fence_barrier_init();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_holder), args.tmem_cols);
    tmem_relinquish();
  }
  fence_proxy_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_O = *tmem_holder;                     // nv blocks of Hp columns
  const uint32_t tmem_S = tmem_O + nv_max * Hp;             // two buffers of `items` blocks of 16 columns

  if (warp == 0) {
    // ------------------------------------ producer (the whole warp, one lane issues) ------------------------------------
    if (n_tiles > 0) {
      const bool leader = elect_one();
      if (leader) {
        mbar_expect_tx(smem_u32(q_full), items * k_halves * (kItem * 128));
        for (int i = 0; i < items; ++i) {
          const int head0 = (i / args.per_kv) * args.group + (i % args.per_kv) * kItem;
          for (int c = 0; c < k_halves; ++c)
            tma_load_2d(smem_u32(sQ) + i * kQItem + c * (kItem * 128), &tmQ, smem_u32(q_full), c * 64, q_row * args.H + head0);
        }
      }
      __syncwarp();
      const int bs = args.block_size;
      const int* table = args.block_tables + static_cast<size_t>(b) * args.max_blocks;
      uint32_t unit = 0;
      bool ok = true;
      auto load_tile = [&](const CUtensorMap* tm, int page, int col0, int halves) {
        const int slot = unit % slots;
        ok = mbar_wait(smem_u32(&empty[slot]), ((unit / slots) & 1) ^ 1, abort_flag, args.status, kStatusWaitTimeoutProducer);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) return;
        if (leader) mbar_expect_tx(smem_u32(&full[slot]), halves * kSub);
        __syncwarp();
        tma_load_pages(leader, smem_u32(sRing + slot * kUnit), kSub, tm, smem_u32(&full[slot]), page, bs, col0, halves);
        ++unit;
      };
      int page = tile_page(table, bs, t0 * kTile, len);
      for (int g = 0; g < args.G && ok; ++g) load_tile(&tmK, page, g * args.D, k_halves);
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int next = j + 1 < n_tiles ? tile_page(table, bs, (t0 + j + 1) * kTile, len) : 0;
        for (int g = 0; g < args.G && ok && j + 1 < n_tiles; ++g) load_tile(&tmK, next, g * args.D, k_halves);
        for (int v = 0; v < nv && ok; ++v) load_tile(&tmV, page, (v0 + v) * args.DV, v_halves);
        page = next;
      }
    }
  } else if (warp == 1) {
    // ------------------------------------ MMA issuer (the whole warp, one lane issues) ------------------------------------
    if (n_tiles > 0) {
      constexpr uint32_t IDESC_S = umma_idesc_bf16(kTile, kItem, 0, 0);     // A = K tile K-major, B = Q K-major
      const uint32_t idesc_pv = umma_idesc_bf16(kTile, Hp, 1, 0);           // A = V tile MN-major, B = P^T K-major
      const bool leader = elect_one();
      const uint64_t ring_k = umma_desc_kmajor_sw128(smem_u32(sRing)), ring_v = umma_desc_mnmajor_sw128(smem_u32(sRing), kSub);
      const uint64_t q_desc = umma_desc_kmajor_sw128(smem_u32(sQ)), p_desc = umma_desc_kmajor_sw128(smem_u32(sP));
      const int k_steps = 4 * k_halves;
      uint32_t unit = 0;
      bool ok = true;
      auto wait = [&](uint64_t* bar, uint32_t parity) {
        ok = mbar_wait(smem_u32(bar), parity, abort_flag, args.status, kStatusWaitTimeoutMma);
        ok = __all_sync(0xffffffffu, ok);
      };
      wait(q_full, 0);
      auto next_unit = [&]() {                              // offset of the next tile of the ring in descriptor units, once it is there
        const int slot = unit % slots;
        wait(&full[slot], (unit / slots) & 1);
        tc_fence_after();
        return static_cast<uint64_t>(slot * (kUnit >> 4));
      };
      auto scores = [&](int j) {
        const int sb = j & 1;
        wait(&s_empty[sb], ((j >> 1) & 1) ^ 1);
        for (int g = 0; g < args.G && ok; ++g) {
          const uint64_t ka = ring_k + next_unit();
          if (!ok) return;
          for (int p = 0; p < args.per_kv; ++p) {
            const int i = g * args.per_kv + p;
            const uint64_t qa = q_desc + i * (kQItem >> 4);
            const uint32_t s_tmem = tmem_S + (sb * items + i) * kItem;
#pragma unroll
            for (int k = 0; k < 8; ++k)
              if (k < k_steps)
                umma_f16_ss_warp(leader, s_tmem, ka + (k >> 2) * (kSub >> 4) + (k & 3) * 2,
                                 qa + (k >> 2) * ((kItem * 128) >> 4) + (k & 3) * 2, IDESC_S, k > 0 ? 1u : 0u);
            umma_commit_warp(leader, smem_u32(&s_full[sb * items + i]));
          }
          umma_commit_warp(leader, smem_u32(&empty[unit % slots]));
          ++unit;
        }
      };
      if (ok) scores(0);
      for (int j = 0; j < n_tiles && ok; ++j) {
        if (j + 1 < n_tiles) scores(j + 1);
        if (ok) wait(p_ready, j & 1);
        const uint64_t pa = p_desc + (j & 1) * (p_buf >> 4);
        for (int v = 0; v < nv && ok; ++v) {
          const uint64_t va = ring_v + next_unit();
          if (!ok) break;
#pragma unroll
          for (int k = 0; k < kTile / 16; ++k)
            umma_f16_ss_warp(leader, tmem_O + v * Hp, va + k * ((16 * 128) >> 4), pa + (k >> 2) * (p_sub >> 4) + (k & 3) * 2, idesc_pv,
                             (j > 0 || k > 0) ? 1u : 0u);
          umma_commit_warp(leader, smem_u32(&empty[unit % slots]));
          ++unit;
        }
        if (ok) umma_commit_warp(leader, smem_u32(pv_done));
      }
    }
  } else {
    // ------------------------------------ softmax / epilogue ------------------------------------
    const int ew = warp & 3;
    const int row = ew * 32 + lane;                         // token row of S^T, value row of O^T
    const uint32_t lane_base = static_cast<uint32_t>(ew * 32) << 16;
    for (int h = 0; h < Hp; ++h) sL[h * kTile + row] = 0.f;
    if (row < kMaxHeads) sM[row] = -INFINITY;
    named_bar_sync(1, 128);
    bool ok = true;
    for (int j = 0; j < n_tiles && ok; ++j) {
      const int sb = j & 1;
      const int tok = (t0 + j) * kTile + row;
      const bool valid = tok < len && tok >= first_tok;
      uint8_t* pcol = sP + sb * p_buf + (row >> 6) * p_sub + (row & 7) * 2;
      const int cell = (row & 63) >> 3;
      // the heads' maxima change seldom: first only see whether some score is more than 2^8 above its head's
      bool fine = true;
      for (int i = 0; i < items; ++i) {
        const int head0 = (i / args.per_kv) * args.group + (i % args.per_kv) * kItem;
        const int nh = min(kItem, (i / args.per_kv + 1) * args.group - head0);
        ok = mbar_wait(smem_u32(&s_full[sb * items + i]), (j >> 1) & 1, abort_flag, args.status, kStatusWaitTimeoutEpilogue) && ok;
        tc_fence_after();
        uint32_t sr[kItem];
        tmem_ld_32x32b_x16(tmem_S + (sb * items + i) * kItem + lane_base, sr);
        tmem_ld_wait();
#pragma unroll
        for (int h = 0; h < kItem; ++h)
          if (h < nh) fine = fine && !(valid && __uint_as_float(sr[h]) * args.scale_log2 > sM[head0 + h] + kRescale);
      }
      const bool rescale = !named_bar_and(2, 128, fine);
      if (rescale) {
        for (int i = 0; i < items; ++i) {
          const int head0 = (i / args.per_kv) * args.group + (i % args.per_kv) * kItem;
          const int nh = min(kItem, (i / args.per_kv + 1) * args.group - head0);
          uint32_t sr[kItem];
          tmem_ld_32x32b_x16(tmem_S + (sb * items + i) * kItem + lane_base, sr);
          tmem_ld_wait();
#pragma unroll
          for (int h = 0; h < kItem; ++h)
            if (h < nh) {
              const float w = warp_max(valid ? __uint_as_float(sr[h]) * args.scale_log2 : -INFINITY);
              if (lane == 0) red[ew * kMaxHeads + head0 + h] = w;
            }
        }
        named_bar_sync(1, 128);
        if (row < args.H) {
          const float mx = fmaxf(fmaxf(red[row], red[kMaxHeads + row]), fmaxf(red[2 * kMaxHeads + row], red[3 * kMaxHeads + row]));
          const float m = sM[row];
          const bool grown = mx > m + kRescale;             // or nothing was accumulated yet
          sAlpha[row] = grown ? (m == -INFINITY ? 0.f : ex2(m - mx)) : 1.f;
          if (grown) sM[row] = mx;
        }
        named_bar_sync(1, 128);
        for (int h = 0; h < args.H; ++h) sL[h * kTile + row] *= sAlpha[h];
      }
      for (int i = 0; i < items; ++i) {
        const int head0 = (i / args.per_kv) * args.group + (i % args.per_kv) * kItem;
        const int nh = min(kItem, (i / args.per_kv + 1) * args.group - head0);
        uint32_t sr[kItem];
        tmem_ld_32x32b_x16(tmem_S + (sb * items + i) * kItem + lane_base, sr);
        tmem_ld_wait();
#pragma unroll
        for (int h = 0; h < kItem; ++h)
          if (h < nh) {
            const int head = head0 + h;
            const float p = valid ? ex2(fmaf(__uint_as_float(sr[h]), args.scale_log2, -sM[head])) : 0.f;
            sL[head * kTile + row] += p;
            *reinterpret_cast<__nv_bfloat16*>(pcol + head * 128 + ((cell ^ (head & 7)) << 4)) = __float2bfloat16_rn(p);
          }
      }
      tc_fence_before();
      mbar_arrive(smem_u32(&s_empty[sb]));
      // the previous O^T update has completed: O^T may be touched, and next tile's weights may go where its weights were
      if (j > 0) ok = mbar_wait(smem_u32(pv_done), (j - 1) & 1, abort_flag, args.status, kStatusWaitTimeoutEpilogue) && ok;
      ok = named_bar_and(2, 128, ok);
      if (!ok) break;
      if (j > 0 && rescale) {
        tc_fence_after();
        for (int c = 0; c < nv * Hp; c += 16) {
          uint32_t r[16];
          tmem_ld_32x32b_x16(tmem_O + lane_base + c, r);
          tmem_ld_wait();
#pragma unroll
          for (int h = 0; h < 16; ++h) {
            const int head = c % Hp + h;
            r[h] = __float_as_uint(__uint_as_float(r[h]) * (head < args.H ? sAlpha[head] : 0.f));
          }
          tmem_st_32x32b_x16(tmem_O + lane_base + c, r);
        }
        tmem_st_wait();
      }
      fence_proxy_async_smem();
      tc_fence_before();
      mbar_arrive(smem_u32(p_ready));
    }
    if (ok && n_tiles > 0) {
      ok = mbar_wait(smem_u32(pv_done), (n_tiles - 1) & 1, abort_flag, args.status, kStatusWaitTimeoutEpilogue);
      ok = named_bar_and(2, 128, ok);
    }
    named_bar_sync(1, 128);
    const bool have = ok && n_tiles > 0;
    if (v0 == 0)
      for (int h = ew; h < args.H; h += 4) {
        const float* l = sL + h * kTile;
        const float sum = warp_sum((l[lane] + l[lane + 32]) + (l[lane + 64] + l[lane + 96]));
        if (lane == 0) {
          float* ml = args.part_ml + ((static_cast<size_t>(b) * args.H + h) * args.splits + split) * 2;
          ml[0] = have ? sM[h] : -INFINITY;
          ml[1] = have ? sum : 0.f;
        }
      }
    if (have) tc_fence_after();
    for (int v = 0; v < nv; ++v)
      for (int c = 0; c < Hp; c += 16) {
        uint32_t r[16];
        if (have) {
          tmem_ld_32x32b_x16(tmem_O + lane_base + v * Hp + c, r);
          tmem_ld_wait();
        }
#pragma unroll
        for (int h = 0; h < 16; ++h)
          if (c + h < args.H && row < args.DV)              // a split without tokens writes zeros, which the merge weighs by zero
            args.part_acc[(((static_cast<size_t>(b) * args.H + c + h) * args.G + v0 + v) * args.splits + split) * args.DV + row] =
                have ? __uint_as_float(r[h]) : 0.f;
      }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_O, args.tmem_cols);
  }
}

constexpr int kParts = 8, kAcc = 8;      // heads g in up to this many parts; result heads at a time

// CTA (key / value head and eight of its result heads, sequence): threads (four columns of the head, part of the heads g)
__global__ void __launch_bounds__(256)
talk_combine_kernel(const float* __restrict__ part_acc, const float* __restrict__ part_ml, const float* __restrict__ talk,
                    const __nv_bfloat16* __restrict__ gate, long long ld_gate, __nv_bfloat16* __restrict__ out, int H, int G, int DV,
                    int splits, int blocks, const int* __restrict__ cu_q) {
  extern __shared__ __align__(16) float sh[];        // [parts][kAcc][DV] partial sums, [H][splits] weights
  const int b = blockIdx.y, kv = blockIdx.x / blocks, group = H / G;
  const int h0 = kv * group + (blockIdx.x % blocks) * kAcc, n = min(kAcc, kv * group + group - h0);
  long long row = b;
  if (cu_q) {
    row = cu_q[b];
    if (cu_q[b + 1] - cu_q[b] != 1) return;
  }
  const int nv = DV / 4, parts = blockDim.x / nv;
  float* sO = sh;
  float* sW = sh + parts * kAcc * DV;
  for (int g = threadIdx.x; g < H; g += blockDim.x) {
    const float* ml = part_ml + (static_cast<size_t>(b) * H + g) * splits * 2;
    float M = -INFINITY, L = 0.f;
    for (int s = 0; s < splits; ++s)
      if (ml[2 * s + 1] > 0.f) M = fmaxf(M, ml[2 * s]);
    for (int s = 0; s < splits; ++s) {
      const float w = ml[2 * s + 1] > 0.f ? exp2f(ml[2 * s] - M) : 0.f;
      sW[g * splits + s] = w;
      L += w * ml[2 * s + 1];
    }
    const float inv = L > 0.f ? 1.f / L : 0.f;
    for (int s = 0; s < splits; ++s) sW[g * splits + s] *= inv;
  }
  __syncthreads();
  const int d = (threadIdx.x % nv) * 4, part = threadIdx.x / nv;
  if (part < parts) {
    float acc[kAcc][4] = {};
    for (int g = part; g < H; g += parts) {
      const float* src = part_acc + ((static_cast<size_t>(b) * H + g) * G + kv) * splits * DV + d;
      float v[4] = {};
#pragma unroll 4
      for (int s = 0; s < splits; ++s) {
        const float4 x = *reinterpret_cast<const float4*>(src + s * DV);
        const float w = sW[g * splits + s];
        v[0] = fmaf(w, x.x, v[0]);
        v[1] = fmaf(w, x.y, v[1]);
        v[2] = fmaf(w, x.z, v[2]);
        v[3] = fmaf(w, x.w, v[3]);
      }
#pragma unroll
      for (int i = 0; i < kAcc; ++i)
        if (i < n) {
          const float t = talk[(h0 + i) * H + g];
#pragma unroll
          for (int e = 0; e < 4; ++e) acc[i][e] = fmaf(t, v[e], acc[i][e]);
        }
    }
#pragma unroll
    for (int i = 0; i < kAcc; ++i)
      if (i < n) *reinterpret_cast<float4*>(sO + (part * kAcc + i) * DV + d) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
  }
  __syncthreads();
  for (int i = threadIdx.x; i < n * DV; i += blockDim.x) {
    float v = 0.f;
    for (int p = 0; p < parts; ++p) v += sO[(p * kAcc + i / DV) * DV + i % DV];
    const long long col = (long long)(h0 + i / DV) * DV + i % DV;
    if (gate) v /= 1.f + __expf(-__bfloat162float(gate[row * ld_gate + col]));
    out[row * H * DV + col] = __float2bfloat16_rn(v);
  }
}

// fills in the shape-dependent part; false when the shapes are not served
bool plan(Args& a, int H, int G, int D, int DV, int block_size) {
  if (G < 1 || H < 1 || H % G || D < 8 || DV < 8 || D > 128 || DV > 128 || D % 8 || DV % 8) return false;
  if (block_size != 16 && block_size != 32 && block_size != 64 && block_size != 128) return false;
  a.H = H; a.G = G; a.group = H / G; a.D = D; a.DV = DV; a.block_size = block_size;
  a.per_kv = (a.group + kItem - 1) / kItem;
  a.items = G * a.per_kv;
  a.Hp = (H + 15) / 16 * 16;
  if (a.items > kMaxItems || a.Hp > kMaxHeads) return false;
  const int left = 512 - 2 * a.items * kItem;
  a.nv = left / a.Hp < G ? left / a.Hp : G;
  if (a.nv < 1) return false;
  const int cols = a.nv * a.Hp + 2 * a.items * kItem;
  a.tmem_cols = 32;
  while (a.tmem_cols < cols) a.tmem_cols *= 2;
  a.slots = (kSmemLimit - fixed_bytes(a.Hp, a.items)) / kUnit;
  if (a.slots > kMaxSlots) a.slots = kMaxSlots;
  return a.slots >= 2;
}

}  // namespace ptd
}  // namespace mfb

extern "C" {
using namespace mfb;

int mfb_paged_talk_decode_supported(int H, int G, int D, int DV, int block_size) {
  ptd::Args a;
  return ptd::plan(a, H, G, D, DV, block_size) ? 1 : 0;
}

// Splits of sequences with up to max_len visible tokens that fill the GPU for `rows` sequences.
int mfb_paged_talk_decode_splits(int rows, int max_len) {
  const int tiles = (max_len + ptd::kTile - 1) / ptd::kTile;
  int best = 1;
  long long best_cost = -1;
  for (int s = 1; s <= tiles && s <= 32; ++s) {
    const long long waves = ((long long)rows * s + 147) / 148;
    const long long cost = waves * (2 * ((tiles + s - 1) / s) + 1) + s / 8;
    if (best_cost < 0 || cost < best_cost) { best_cost = cost; best = s; }
  }
  return best;
}

long long mfb_paged_talk_decode_scratch_bytes(int B, int H, int G, int DV, int splits) {
  return (long long)B * H * splits * ((long long)G * DV + 2) * 4;
}

// q [rows, H, D], caches [num_blocks, block_size, G, D | DV], gate [rows, H DV] (rows ld_gate apart) or null, out [rows, H, DV], all
// bf16; talk [H, H] fp32. cu_q null: row b belongs to sequence b (rows == B); else [B + 1] row boundaries of a ragged batch, of which
// only the sequences with one row are computed and written. window > 0: the last `window` keys only.
int mfb_paged_talk_decode(const void* q, const void* key_cache, const void* value_cache, const int* block_tables,
                          const int* context_lens, const int* cu_q, const float* talk, const void* gate, long long ld_gate, void* out,
                          void* scratch, int splits, int rows, int B, int H, int G, int D, int DV, int num_blocks, int block_size,
                          int max_blocks, int window, float scale, int* status, cudaStream_t stream) {
  ptd::Args a;
  if (!ptd::plan(a, H, G, D, DV, block_size) || splits < 1 || splits > 32 || num_blocks < 1 || (!cu_q && rows != B)) {
    mfb_host::set_error("paged_talk_decode: H=%d G=%d D=%d DV=%d block_size=%d splits=%d", H, G, D, DV, block_size, splits);
    return 1;
  }
  if (B <= 0 || rows <= 0) return 0;
  CUtensorMap tQ, tK, tV;
  int rc;
  const CUtensorMapDataType BF = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  const uint64_t n = (uint64_t)num_blocks * block_size, kp = (uint64_t)G * D, vp = (uint64_t)G * DV;
  if ((rc = mfb_host::make_tmap_2d(&tQ, q, 2, BF, (uint64_t)rows * H, D, D, ptd::kItem, 64))) return 20 + rc;
  if ((rc = mfb_host::make_tmap_2d(&tK, key_cache, 2, BF, n, kp, kp, block_size, 64))) return 30 + rc;
  if ((rc = mfb_host::make_tmap_2d(&tV, value_cache, 2, BF, n, vp, vp, block_size, 64))) return 40 + rc;
  a.block_tables = block_tables; a.context_lens = context_lens; a.cu_q = cu_q; a.max_blocks = max_blocks; a.splits = splits;
  a.window = window; a.scale_log2 = scale * 1.4426950408889634f; a.status = status;
  a.part_acc = reinterpret_cast<float*>(scratch);
  a.part_ml = a.part_acc + (size_t)B * H * G * splits * DV;
  if (reinterpret_cast<uintptr_t>(scratch) & 15) {
    mfb_host::set_error("paged_talk_decode: the scratch must start on 16 bytes");
    return 1;
  }
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(ptd::paged_talk_decode_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, ptd::kSmemLimit) != cudaSuccess ||
        cudaFuncSetAttribute(ptd::talk_combine_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024) != cudaSuccess) {
      mfb_host::set_error("paged_talk_decode: cannot raise the shared memory limit");
      return 10;
    }
    attr_set = true;
  }
  const int smem = ptd::fixed_bytes(a.Hp, a.items) + a.slots * ptd::kUnit;
  ptd::paged_talk_decode_kernel<<<dim3(splits, (G + a.nv - 1) / a.nv, B), ptd::kThreads, smem, stream>>>(tQ, tK, tV, a);
  if (cudaGetLastError() != cudaSuccess) { mfb_host::set_error("paged_talk_decode: launch failed"); return 11; }
  const int blocks = (H / G + ptd::kAcc - 1) / ptd::kAcc;
  const int nv = DV / 4, parts = 256 / nv < ptd::kParts ? 256 / nv : ptd::kParts;
  const int threads = (parts * nv + 31) / 32 * 32;
  const size_t csmem = ((size_t)H * splits + (size_t)(threads / nv) * ptd::kAcc * DV) * 4;
  ptd::talk_combine_kernel<<<dim3(G * blocks, B), threads, csmem, stream>>>(
      a.part_acc, a.part_ml, talk, (const __nv_bfloat16*)gate, ld_gate, (__nv_bfloat16*)out, H, G, DV, splits, blocks, cu_q);
  return cudaGetLastError() == cudaSuccess ? 0 : 12;
}

}  // extern "C"
