// Decode attention over a paged cache of latents, keys and values at once (sm_100a, tcgen05 + TMA), with an optional sliding
// window and softmax sink. The factors that make keys and values of a latent are absorbed into query and result, so that one
// decode step is, per sequence and head h with q, c of `rank` numbers (a multiple of 8 up to 576), of which the first `v_rank` (up to
// 512) make the values and the others only keys (a key part with positions, shared by the heads):
//     s[t]   = scale * <q[h], c[t]>                       max(0, len - window) <= t < len
//     o[h,:] = sum_t softmax(s)[t] * c[t][:v_rank]        the sink is one more term of the softmax's denominator
// As in mla_decode.cu, which serves one fixed latent width beside rotated columns, the products are transposed so that the tokens
// fill the 128 rows of the tensor core, and a CTA takes (split of the sequence, 16 or 32 heads, sequence):
//     S^T [128 tokens x heads]       = C_tile (A, K-major) . Q^T (B, K-major)
//     O^T [rank x heads]            += C_tile^T (A, MN-major: the same bytes) . P^T [heads x 128 tokens] (B, K-major)
// A tile of 128 tokens lies in up to five 32 KB slots of a ring (128 latent columns each, the last one possibly half) from its
// scores to its last product, so the cache is read once per 32 heads. Where two tiles fit the ring, the scores of the next tile
// are computed under the softmax of this one. Columns past the rank are zero fill in both operands; the rows of O^T that belong
// to them are not stored.
//
// Roles (192 threads): warp 0 TMA producer (block-table lookups), warp 1 MMA issuer + TMEM owner, warps 2..5 softmax / rescale /
// epilogue. Every wait is bounded (common.cuh). The splits are merged by the combine kernel of paged_attention.cu.
#include "common.cuh"

namespace mfb {
namespace latd {

constexpr int kThreads = 192;
constexpr int kTile = 128;              // tokens per tile
constexpr int kMaxRank = 576, kMaxVRank = 512;
constexpr int kSub = kTile * 128;       // [128 tokens][64 columns] swizzled sub-tile, 16 KB
constexpr int kUnit = 2 * kSub;         // ring slot: a pair of sub-tiles (128 columns)
constexpr int kMaxSlots = 6;
constexpr float kRescale = 8.0f;

// per number of heads of a CTA: P^T as two [heads][64 tokens] K-major sub-tiles, Q as [heads][64 columns] sub-tiles
template <int HEADS>
struct Shape {
  static constexpr int kPBytes = 2 * HEADS * 128, kQSub = HEADS * 128, kQBytes = kMaxRank / 64 * kQSub;
  static constexpr int kFixed = kPBytes + kQBytes + 4 * HEADS * 4 + (7 + 2 * kMaxSlots) * 8 + 16 + 1024;
  static constexpr int kFit = (232448 - kFixed) / kUnit;
  static constexpr int kSlots = kFit < kMaxSlots ? kFit : kMaxSlots;
  static constexpr int kSmem = kFixed + kSlots * kUnit;
  static constexpr int kTmemCols = HEADS <= 16 ? 128 : 256;      // four blocks of O^T and two buffers of S^T
};

struct Args {
  const int* block_tables;   // [B, max_blocks]
  const int* context_lens;   // [B]
  int max_blocks, block_size, num_heads, splits, rank, v_rank, window;
  float scale_log2;
  float* part_o;             // [B, num_heads, splits, v_rank] unnormalised
  float* part_ml;            // [B, num_heads, splits, 2]: running max (log2 units), sum
  int* status;
};

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm volatile("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

template <int HEADS>
__global__ void __launch_bounds__(kThreads, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmC, const Args args) {
  using Sh = Shape<HEADS>;
  constexpr int kHeads = HEADS, kSlots = Sh::kSlots, kPBytes = Sh::kPBytes, kQSub = Sh::kQSub, kQBytes = Sh::kQBytes;
  constexpr int kTmemCols = Sh::kTmemCols;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) &
                                             ~static_cast<uintptr_t>(1023));
  uint8_t* sRing = smem;
  uint8_t* sP = sRing + kSlots * kUnit;
  uint8_t* sQ = sP + kPBytes;
  float* red = reinterpret_cast<float*>(sQ + kQBytes);  // [4 warps][heads]
  uint64_t* bars = reinterpret_cast<uint64_t*>(red + 4 * kHeads);
  uint64_t* q_full = bars;                  // 1
  uint64_t* p_ready = bars + 1;             // 1
  uint64_t* pv_done = bars + 2;             // 1
  uint64_t* s_full = bars + 3;              // 2
  uint64_t* s_empty = bars + 5;             // 2
  uint64_t* full = bars + 7;                // kSlots
  uint64_t* empty = full + kMaxSlots;       // kSlots
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(empty + kMaxSlots);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_holder + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int split = blockIdx.x, chunk = blockIdx.y, b = blockIdx.z;
  const int len = args.context_lens[b];
  const int first_tok = args.window > 0 && len > args.window ? len - args.window : 0;
  const int base_tile = first_tok / kTile;
  const int n_tiles_all = (len + kTile - 1) / kTile - base_tile;
  const int per = (n_tiles_all + args.splits - 1) / args.splits;
  const int rel0 = split * per;
  const int rel1 = (rel0 + per < n_tiles_all) ? rel0 + per : n_tiles_all;
  const int n_tiles = rel1 > rel0 ? rel1 - rel0 : 0;
  const int t0 = base_tile + rel0;
  const int head0 = chunk * kHeads;
  const int subs = (args.rank + 63) / 64, units = (subs + 1) / 2;      // 64-column sub-tiles, pairs of them
  const int v_units = (args.v_rank + 127) / 128;                       // pairs that hold values

  if (threadIdx.x == 0) {
    *abort_flag = 0;
    mbar_init(smem_u32(q_full), 1);
    for (int s = 0; s < kSlots; ++s) {
      mbar_init(smem_u32(&full[s]), 1);
      mbar_init(smem_u32(&empty[s]), 1);
    }
    for (int s = 0; s < 2; ++s) {
      mbar_init(smem_u32(&s_full[s]), 1);
      mbar_init(smem_u32(&s_empty[s]), 128);
    }
    mbar_init(smem_u32(p_ready), 128);
    mbar_init(smem_u32(pv_done), 1);
    fence_barrier_init();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmC);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_holder), kTmemCols);
    tmem_relinquish();
  }
  fence_proxy_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_holder;
  const uint32_t tmem_O = tmem_base;                   // 4 blocks of `heads` columns
  const uint32_t tmem_S = tmem_base + 4 * kHeads;      // 2 buffers of `heads` columns

  if (warp == 0) {
    // ------------------------------------ producer (the whole warp, one lane issues) ------------------------------------
    if (n_tiles > 0) {
      const bool leader = elect_one();
      if (leader) {
        mbar_expect_tx(smem_u32(q_full), subs * kQSub);
        for (int c = 0; c < subs; ++c) tma_load_2d(smem_u32(sQ) + c * kQSub, &tmQ, smem_u32(q_full), c * 64, b * args.num_heads + head0);
      }
      __syncwarp();
      const int bs = args.block_size;
      const int* table = args.block_tables + static_cast<size_t>(b) * args.max_blocks;
      uint32_t unit = 0;
      bool ok = true;
      int page = tile_page(table, bs, t0 * kTile, len);
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int next = j + 1 < n_tiles ? tile_page(table, bs, (t0 + j + 1) * kTile, len) : 0;
        for (int pair = 0; pair < units && ok; ++pair) {
          const int slot = unit % kSlots;
          ok = mbar_wait(smem_u32(&empty[slot]), ((unit / kSlots) & 1) ^ 1, abort_flag, args.status, kStatusWaitTimeoutProducer);
          ok = __all_sync(0xffffffffu, ok);
          if (!ok) break;
          const int two = 2 * pair + 1 < subs ? 2 : 1;
          if (leader) mbar_expect_tx(smem_u32(&full[slot]), two * kSub);
          __syncwarp();
          tma_load_pages(leader, smem_u32(sRing + slot * kUnit), kSub, &tmC, smem_u32(&full[slot]), page, bs, pair * 128, two);
          ++unit;
        }
        page = next;
      }
    }
  } else if (warp == 1) {
    // ------------------------------------ MMA issuer (the whole warp, one lane issues) ------------------------------------
    if (n_tiles > 0) {
      constexpr uint32_t IDESC_S = umma_idesc_bf16(kTile, kHeads, 0, 0);   // A = cache K-major, B = Q K-major
      constexpr uint32_t IDESC_PV = umma_idesc_bf16(kTile, kHeads, 1, 0);  // A = cache MN-major, B = P^T K-major
      const bool leader = elect_one();
      const uint64_t ring_k = umma_desc_kmajor_sw128(smem_u32(sRing)), ring_v = umma_desc_mnmajor_sw128(smem_u32(sRing), kSub);
      const uint64_t q_desc = umma_desc_kmajor_sw128(smem_u32(sQ)), p_desc = umma_desc_kmajor_sw128(smem_u32(sP));
      bool ok = true;
      auto wait = [&](uint64_t* bar, uint32_t parity) {
        ok = mbar_wait(smem_u32(bar), parity, abort_flag, args.status, kStatusWaitTimeoutMma);
        ok = __all_sync(0xffffffffu, ok);
      };
      // ---- S^T(j) = C . Q^T over the pairs of the tile, which stay in the ring ----
      auto scores = [&](int j) {
        const int sb = j & 1;
        wait(&s_empty[sb], ((j >> 1) & 1) ^ 1);
        for (int u = 0; u < units && ok; ++u) {
          const int unit = j * units + u, slot = unit % kSlots;
          wait(&full[slot], (unit / kSlots) & 1);
          if (!ok) return;
          tc_fence_after();
          const uint64_t ca = ring_k + slot * (kUnit >> 4), qa = q_desc + 2 * u * (kQSub >> 4);
          const int ksteps = 2 * u + 1 < subs ? 8 : 4;
#pragma unroll
          for (int k = 0; k < 8; ++k)
            if (k < ksteps)
              umma_f16_ss_warp(leader, tmem_S + sb * kHeads, ca + (k >> 2) * (kSub >> 4) + (k & 3) * 2,
                               qa + (k >> 2) * (kQSub >> 4) + (k & 3) * 2, IDESC_S, (u > 0 || k > 0) ? 1u : 0u);
        }
        if (ok) umma_commit_warp(leader, smem_u32(&s_full[sb]));
      };
      wait(q_full, 0);
      const bool ahead = 2 * units <= kSlots;
      if (ok && ahead) scores(0);
      for (int j = 0; j < n_tiles && ok; ++j) {
        if (!ahead) scores(j);
        else if (j + 1 < n_tiles) scores(j + 1);
        // ---- O^T += C^T(j) . P^T(j) ----
        if (ok) wait(p_ready, j & 1);
        if (!ok) break;
        tc_fence_after();
        for (int m = 0; m < units; ++m) {
          const int slot = (j * units + m) % kSlots;
          const uint64_t ca = ring_v + slot * (kUnit >> 4);
          if (m < v_units) {
#pragma unroll
            for (int k = 0; k < kTile / 16; ++k)
              umma_f16_ss_warp(leader, tmem_O + m * kHeads, ca + k * ((16 * 128) >> 4), p_desc + (k >> 2) * ((kHeads * 128) >> 4) + (k & 3) * 2,
                               IDESC_PV, (j > 0 || k > 0) ? 1u : 0u);
          }
          umma_commit_warp(leader, smem_u32(&empty[slot]));
        }
        umma_commit_warp(leader, smem_u32(pv_done));
      }
    }
  } else {
    // ------------------------------------ softmax / epilogue ------------------------------------
    const int ew = warp & 3;
    const int row = ew * 32 + lane;                 // token row of S^T, dv row of O^T
    const uint32_t lane_base = static_cast<uint32_t>(ew * 32) << 16;
    float m_used[kHeads], l_part[kHeads];
#pragma unroll
    for (int h = 0; h < kHeads; ++h) { m_used[h] = -INFINITY; l_part[h] = 0.f; }
    bool ok = true;
    for (int j = 0; j < n_tiles; ++j) {
      const int sb = j & 1;
      const uint32_t sph = (j >> 1) & 1;
      ok = mbar_wait(smem_u32(&s_full[sb]), sph, abort_flag, args.status, kStatusWaitTimeoutEpilogue);
      ok = named_bar_and(2, 128, ok);
      if (!ok) break;
      tc_fence_after();
      uint32_t sr[kHeads];
#pragma unroll
      for (int c = 0; c < kHeads; c += 16)
        tmem_ld_32x32b_x16(tmem_S + sb * kHeads + c + lane_base, *reinterpret_cast<uint32_t(*)[16]>(&sr[c]));
      tmem_ld_wait();
      tc_fence_before();
      mbar_arrive(smem_u32(&s_empty[sb]));
      float s[kHeads];
      const int tok = (t0 + j) * kTile + row;
      const bool valid = tok < len && tok >= first_tok;
#pragma unroll
      for (int h = 0; h < kHeads; ++h) s[h] = valid ? __uint_as_float(sr[h]) * args.scale_log2 : -INFINITY;
      // the heads' maxima change seldom: first only see whether some score is more than 2^8 above its head's
      bool fine = true;
#pragma unroll
      for (int h = 0; h < kHeads; ++h) fine = fine && !(s[h] > m_used[h] + kRescale);
      const bool any_rescale = !named_bar_and(3, 128, fine);
      float alpha[kHeads];
#pragma unroll
      for (int h = 0; h < kHeads; ++h) alpha[h] = 1.f;
      if (any_rescale) {
        // per-head maximum over the 128 tokens of the tile
#pragma unroll
        for (int h = 0; h < kHeads; ++h) {
          const float w = warp_max(s[h]);
          if (lane == 0) red[ew * kHeads + h] = w;
        }
        named_bar_sync(1, 128);
#pragma unroll
        for (int h = 0; h < kHeads; ++h) {
          const float mx = fmaxf(fmaxf(red[h], red[kHeads + h]), fmaxf(red[2 * kHeads + h], red[3 * kHeads + h]));
          if (mx > m_used[h] + kRescale) {              // or nothing was accumulated yet
            alpha[h] = m_used[h] == -INFINITY ? 0.f : ex2(m_used[h] - mx);
            m_used[h] = mx;
          }
        }
      }
#pragma unroll
      for (int h = 0; h < kHeads; ++h) {
        const float neg_m = (m_used[h] == -INFINITY) ? 0.f : -m_used[h];
        s[h] = valid ? ex2(s[h] + neg_m) : 0.f;
        l_part[h] = l_part[h] * alpha[h] + s[h];
      }
      if (j > 0) {
        // the previous O^T update has completed: P^T may be overwritten and O^T touched
        ok = mbar_wait(smem_u32(pv_done), (j - 1) & 1, abort_flag, args.status, kStatusWaitTimeoutEpilogue);
        if (ok && any_rescale) {
          tc_fence_after();
          for (int m = 0; m < v_units; ++m)
#pragma unroll
            for (int c = 0; c < kHeads; c += 16) {
              uint32_t r[16];
              tmem_ld_32x32b_x16(tmem_O + lane_base + m * kHeads + c, r);
              tmem_ld_wait();
#pragma unroll
              for (int h = 0; h < 16; ++h) r[h] = __float_as_uint(__uint_as_float(r[h]) * alpha[c + h]);
              tmem_st_32x32b_x16(tmem_O + lane_base + m * kHeads + c, r);
            }
          tmem_st_wait();
        }
      }
      ok = named_bar_and(2, 128, ok);               // also orders the reads of `red` before the next tile's writes
      if (!ok) break;
      // P^T[h][token] as a K-major operand: sub-tile of 64 tokens, row h of 128 bytes, 16-byte chunks swizzled by row
      {
        uint8_t* pcol = sP + (row >> 6) * (kHeads * 128) + (row & 7) * 2;
        const int chunk = (row & 63) >> 3;
#pragma unroll
        for (int h = 0; h < kHeads; ++h)
          *reinterpret_cast<__nv_bfloat16*>(pcol + h * 128 + ((chunk ^ (h & 7)) << 4)) = __float2bfloat16_rn(s[h]);
      }
      fence_proxy_async_smem();
      tc_fence_before();
      mbar_arrive(smem_u32(p_ready));
    }
    if (ok && n_tiles > 0) {
      ok = mbar_wait(smem_u32(pv_done), (n_tiles - 1) & 1, abort_flag, args.status, kStatusWaitTimeoutEpilogue);
      ok = named_bar_and(2, 128, ok);
    }
    // per-head sums over the 128 token rows
    float l_tot[kHeads];
#pragma unroll
    for (int h = 0; h < kHeads; ++h) {
      const float w = warp_sum(l_part[h]);
      if (lane == 0) red[ew * kHeads + h] = w;
    }
    named_bar_sync(1, 128);
#pragma unroll
    for (int h = 0; h < kHeads; ++h)
      l_tot[h] = (red[h] + red[kHeads + h]) + (red[2 * kHeads + h] + red[3 * kHeads + h]);
    const bool have = ok && n_tiles > 0;
    const size_t first_row = static_cast<size_t>(b) * args.num_heads + head0;
    if (row < kHeads && head0 + row < args.num_heads) {
      float mh = -INFINITY, lh = 0.f;
#pragma unroll
      for (int h = 0; h < kHeads; ++h)
        if (h == row) { mh = m_used[h]; lh = l_tot[h]; }
      if (!have) { mh = -INFINITY; lh = 0.f; }
      float* ml = args.part_ml + ((first_row + row) * args.splits + split) * 2;
      ml[0] = mh;
      ml[1] = lh;
    }
    if (have) tc_fence_after();
    for (int m = 0; m < v_units; ++m) {
      const int col = m * 128 + row;
#pragma unroll
      for (int c = 0; c < kHeads; c += 16) {
        uint32_t r[16];
        if (have) {
          tmem_ld_32x32b_x16(tmem_O + lane_base + m * kHeads + c, r);
          tmem_ld_wait();
        }
#pragma unroll
        for (int h = 0; h < 16; ++h)
          if (head0 + c + h < args.num_heads && col < args.v_rank)    // a split without tokens writes zeros, which the merge weighs by zero
            args.part_o[((first_row + c + h) * args.splits + split) * args.v_rank + col] = have ? __uint_as_float(r[h]) : 0.f;
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, kTmemCols);
  }
}


template <int HEADS>
int launch(const CUtensorMap& tQ, const CUtensorMap& tC, const Args& a, int B, cudaStream_t stream) {
  using Sh = Shape<HEADS>;
  static_assert(Sh::kSlots >= (kMaxRank + 127) / 128, "a tile lies in the ring as a whole");
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(latent_decode_kernel<HEADS>, cudaFuncAttributeMaxDynamicSharedMemorySize, Sh::kSmem) != cudaSuccess) {
      mfb_host::set_error("latent_decode: cannot raise shared memory limit");
      return 10;
    }
    attr_set = true;
  }
  const dim3 grid(a.splits, (a.num_heads + HEADS - 1) / HEADS, B);
  latent_decode_kernel<HEADS><<<grid, kThreads, Sh::kSmem, stream>>>(tQ, tC, a);
  if (cudaGetLastError() != cudaSuccess) { mfb_host::set_error("latent_decode: launch failed"); return 11; }
  return 0;
}

int heads_per_cta(int num_heads) { return num_heads > 16 ? 32 : 16; }

}  // namespace latd
}  // namespace mfb

extern "C" {
using namespace mfb;

int mfb_paged_combine_ex(const float* part_acc, const float* part_ml, void* out, int splits, int rows, int hd, int Hq,
                         const int* cu_q, const float* sink, long long ld_out, float out_scale,
                         cudaStream_t stream);      // paged_attention.cu

int mfb_latent_decode_supported(int rank, int v_rank, int block_size) {
  return v_rank >= 8 && v_rank <= latd::kMaxVRank && v_rank % 8 == 0 && rank >= v_rank && rank <= latd::kMaxRank && rank % 8 == 0 &&
                 (block_size == 16 || block_size == 32 || block_size == 64 || block_size == 128)
             ? 1 : 0;
}

// Number of sequence splits that fills the GPU for a batch of B sequences of up to max_len visible tokens.
int mfb_latent_decode_splits(int B, int num_heads, int max_len) {
  // cost of a choice = waves of CTAs over the 148 SMs x (tiles per CTA + about one tile of fixed work per CTA)
  const int per = latd::heads_per_cta(num_heads), chunks = (num_heads + per - 1) / per;
  const int tiles = (max_len + latd::kTile - 1) / latd::kTile;
  int best = 1;
  long long best_cost = -1;
  for (int s = 1; s <= tiles && s <= 32; ++s) {
    const long long ctas = static_cast<long long>(B) * chunks * s;
    const long long waves = (ctas + 147) / 148;
    const long long cost = waves * ((tiles + s - 1) / s + 1);
    if (best_cost < 0 || cost < best_cost) { best_cost = cost; best = s; }
  }
  return best;
}

long long mfb_latent_decode_scratch_bytes(int B, int num_heads, int v_rank, int splits) {
  return static_cast<long long>(B) * splits * num_heads * (v_rank + 2) * 4;
}

// q [B, num_heads, rank] (queries in latent space), cache [num_blocks, block_size, rank], out [B, num_heads, v_rank], all bf16;
// block_tables [B, max_blocks]; context_lens [B] counts the tokens in the cache, the new one included; window > 0: only the last
// `window` of them; sink [num_heads] fp32 or null; scratch: mfb_latent_decode_scratch_bytes.
int mfb_latent_decode(const void* q, const void* cache, const int* block_tables, const int* context_lens, const float* sink, void* out,
                      void* scratch, int splits, int B, int num_heads, int rank, int v_rank, int num_blocks, int block_size, int max_blocks,
                      int window, float scale, int* status, cudaStream_t stream) {
  if (!mfb_latent_decode_supported(rank, v_rank, block_size) || num_heads < 1 || splits < 1 || num_blocks < 1 || max_blocks < 1) {
    mfb_host::set_error("latent_decode: heads=%d rank=%d v_rank=%d splits=%d block_size=%d", num_heads, rank, v_rank, splits, block_size);
    return 1;
  }
  if (B <= 0) return 0;
  CUtensorMap tQ, tC;
  int rc;
  const CUtensorMapDataType BF = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  if ((rc = mfb_host::make_tmap_2d(&tQ, q, 2, BF, (uint64_t)B * num_heads, rank, rank, latd::heads_per_cta(num_heads), 64))) return 20 + rc;
  if ((rc = mfb_host::make_tmap_2d(&tC, cache, 2, BF, (uint64_t)num_blocks * block_size, rank, rank, block_size, 64))) return 30 + rc;
  latd::Args a;
  a.block_tables = block_tables; a.context_lens = context_lens; a.max_blocks = max_blocks; a.block_size = block_size;
  a.num_heads = num_heads; a.splits = splits; a.rank = rank; a.v_rank = v_rank; a.window = window; a.scale_log2 = scale * 1.4426950408889634f;
  a.part_o = reinterpret_cast<float*>(scratch);
  a.part_ml = a.part_o + static_cast<size_t>(B) * splits * num_heads * v_rank;
  a.status = status;
  rc = latd::heads_per_cta(num_heads) == 32 ? latd::launch<32>(tQ, tC, a, B, stream) : latd::launch<16>(tQ, tC, a, B, stream);
  if (rc) return rc;
  return mfb_paged_combine_ex(a.part_o, a.part_ml, out, splits, B * num_heads, v_rank, num_heads, nullptr, sink,
                              (long long)num_heads * v_rank, 1.f, stream);
}

}  // extern "C"
