// Absorbed latent attention of single query rows on the tensor cores (tcgen05): every head of a row attends to the same
// cache rows, [latent | rotated key part], and the values are the latent part of the rows themselves.
//
// A tile of 128 cache rows is fetched once and used twice:
//     S^T [keys x heads]       = K Q^T      A = the tile, K-major; B = the absorbed queries, 16 or 32 heads
//     O^T [latent x heads]    += C^T P^T    A = the same tile read MN-major, 128 latent columns per MMA block
// so M is always full although a token has few query rows, and the kernel is bound by the cache bytes: the tile's
// columns travel as pairs of 64-column chunks with a barrier each, the score product starts with the first pair and a
// pair is refilled as soon as its part of O^T is done; the next tile travels to L2 meanwhile, since wide rows leave
// room for one tile in shared memory (two tiles of 64 keys were 40 % slower: an MMA of this shape takes about 60 cycles
// whether it has 64 or 128 rows). Rows of up to 640 elements, latents of up to 512. The keys of a
// row can be cut into splits, whose fp32 partial results a second kernel merges. Under a sliding window only the tiles that
// hold visible keys are visited; a sink per head joins the denominator at the end. EXACT: the softmax weights reach the
// product with the latents as two bf16 terms, which keeps 16 bits of them.
//
// Roles (192 threads): warp 0 TMA producer, warp 1 MMA issuer, warps 2..5 softmax (one thread per key of the tile),
// rescaling and epilogue (one thread per latent column). Waits are bounded; after a timeout the roles keep their trip
// counts, report TW_ERR_MBAR_TIMEOUT and leave through the tear-down.
#include "tw_elect.cuh"
#include "tw_host.h"
#include "tw_kernels.h"

namespace tw {

constexpr int LD_BN = 128;                       // keys per tile
constexpr int LD_THREADS = 192;
constexpr int LD_MAX_PAIRS = 5, LD_MAX_STAGES = 4;
constexpr int LD_SMEM_LIMIT = 227 * 1024;

struct LatentDecodeParams {
  const __nv_bfloat16* q;        // [n, heads, row]
  __nv_bfloat16* out;            // [n, heads, kv_rank]
  const __nv_bfloat16* cache;    // [blocks, page, row]
  const int *tok_seq, *tok_kvlen, *block_table;
  int max_blocks, page, heads, row, kv_rank, splits, chunks, stages;
  float scale_log2;
  float *part_o, *part_ml;
  uint32_t* status;
  int window;                    // > 0: the last `window` keys are visible
  const float* sink;             // [heads] or null: exp(sink) joins the denominator
};

__device__ __forceinline__ float ld_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void ld_softmax_sync() { asm volatile("bar.sync 1, 128;" ::: "memory"); }
__device__ __forceinline__ void tmem_ld_cols(uint32_t addr, uint32_t (&r)[16]) { tmem_ld_32x16(addr, r); }
__device__ __forceinline__ void tmem_ld_cols(uint32_t addr, uint32_t (&r)[32]) { tmem_ld_32x32(addr, r); }
__device__ __forceinline__ void tmem_st_cols(uint32_t addr, const uint32_t (&r)[16]) { tmem_st_32x16(addr, r); }
__device__ __forceinline__ void tmem_st_cols(uint32_t addr, const uint32_t (&r)[32]) { tmem_st_32x32(addr, r); }

// Shared memory behind the tiles: Q, P, barriers, exchange.
template <int NC, bool EXACT>
__host__ __device__ constexpr int ld_fixed_bytes(int chunks) {
  return chunks * NC * 128 + (EXACT ? 4 : 2) * NC * 128 + 512 + 2 * 4 * NC * 4 + 1024;
}

template <int NC, bool EXACT>
__global__ void __launch_bounds__(LD_THREADS, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmC, const __grid_constant__ CUtensorMap tmQ,
                     const LatentDecodeParams p) {
  constexpr uint32_t IDESC_S = make_idesc_bf16(LD_BN, NC, 0, 0);     // A = rows (K-major), B = Q (K-major)
  constexpr uint32_t IDESC_O = make_idesc_bf16(128, NC, 1, 0);       // A = latent columns (MN-major), B = P (K-major)
  constexpr uint32_t TMEM_COLS = NC == 16 ? 128 : 256;               // 2 NC for S, 4 NC for O
  constexpr uint32_t COL_O = 2 * NC;

  constexpr int CHUNK = LD_BN * 128;                                    // 64 columns of a tile

  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) &
                                             ~static_cast<uintptr_t>(1023));
  const int pairs = (p.chunks + 1) >> 1;
  const int v_chunks = (p.kv_rank + 63) >> 6, v_pairs = (v_chunks + 1) >> 1;
  const int tile_bytes = pairs * 2 * CHUNK;
  uint8_t* s_q = smem + p.stages * tile_bytes;
  uint8_t* s_p = s_q + p.chunks * NC * 128;
  constexpr int P_LO = 2 * NC * 128;                          // second terms of the weights behind the first ones
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_p + (EXACT ? 2 : 1) * P_LO);
  uint64_t* full = bars;                                      // [stages][LD_MAX_PAIRS]
  uint64_t* empty = bars + LD_MAX_STAGES * LD_MAX_PAIRS;
  uint64_t* s_full = bars + 2 * LD_MAX_STAGES * LD_MAX_PAIRS;  // [2]
  uint64_t* p_ready = s_full + 2;
  uint64_t* o_done = s_full + 3;
  uint64_t* q_ready = s_full + 4;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(s_full + 5);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* xchg = reinterpret_cast<float*>(reinterpret_cast<uint8_t*>(bars) + 512);    // [2][4 warps][NC]

  const int warp = threadIdx.x >> 5;
  const int lane = threadIdx.x & 31;
  const int tok = blockIdx.x, h0 = blockIdx.y * NC, split = blockIdx.z;
  const int G = min(NC, p.heads - h0);
  const int seq = p.tok_seq[tok];
  const int kv_len = p.tok_kvlen[tok];
  const int win_lo = p.window > 0 ? max(0, kv_len - p.window) : 0, j_lo = win_lo / LD_BN;
  const int tiles_total = (kv_len + LD_BN - 1) / LD_BN - j_lo;
  const int per_split = (tiles_total + p.splits - 1) / p.splits;
  const int n_tiles = max(0, min(tiles_total - split * per_split, per_split));
  const int t_begin = j_lo + split * per_split;

  if (threadIdx.x == 0) {
    for (int i = 0; i < p.stages * LD_MAX_PAIRS; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    mbar_init(&s_full[0], 1);
    mbar_init(&s_full[1], 1);
    mbar_init(p_ready, 128);
    mbar_init(o_done, 1);
    mbar_init(q_ready, 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 0) {
    // ---------------- TMA producer (uniform over the warp, see the issuer) ----------------
    if (n_tiles > 0) {
      // The queries: NC rows from the token's first head on. Rows behind the block's last head are another token's or
      // zeros; their columns of S and O are not used.
      mbar_expect_tx_e(q_ready, p.chunks * NC * 128);
      for (int c = 0; c < p.chunks; ++c) tma_load_2d_e(s_q + c * NC * 128, &tmQ, q_ready, c * 64, tok * p.heads + h0);
      // a tile is several pages, or a page several tiles; a piece (rows of one page) is contiguous in memory
      const int piece = min(p.page, LD_BN), pieces = LD_BN / piece;
      const int last_page = (kv_len - 1) / p.page;
      const int* table = p.block_table + static_cast<long long>(seq) * p.max_blocks;
      const uint32_t piece_bytes = piece * p.row * 2;
      // A tile's copies are issued when its buffer is free; by then its bytes should not be in DRAM any more.
      auto prefetch = [&](int j) {
        if (j >= n_tiles || lane >= pieces) return;
        const int key = (t_begin + j) * LD_BN + lane * piece;
        if (key >= kv_len) return;
        const __nv_bfloat16* src =
            p.cache + (static_cast<long long>(table[key / p.page]) * p.page + key % p.page) * p.row;
        asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(src), "r"(piece_bytes) : "memory");
      };
      for (int j = 0; j < p.stages; ++j) prefetch(j);
      bool ok = true;
      for (int j = 0; ok && j < n_tiles; ++j) {
        const int st = j % p.stages;
        const uint32_t ph = (j / p.stages) & 1;
        const int key0 = (t_begin + j) * LD_BN;
        // page ids of the tile's pieces, one per lane
        const int block = table[min((key0 + (lane & (pieces - 1)) * piece) / p.page, last_page)];
        uint8_t* tile = smem + st * tile_bytes;
        for (int pr = 0; pr < pairs; ++pr) {
          if (!mbar_wait_warp(&empty[st * LD_MAX_PAIRS + pr], ph ^ 1)) { ok = false; break; }
          uint64_t* bar = &full[st * LD_MAX_PAIRS + pr];
          const bool two = 2 * pr + 1 < p.chunks;
          mbar_expect_tx_e(bar, (two ? 2 : 1) * CHUNK);
          for (int pc = 0; pc < pieces; ++pc) {
            const int blk = __shfl_sync(0xffffffffu, block, pc), y = (key0 + pc * piece) % p.page;
            uint8_t* dst = tile + pr * 2 * CHUNK + pc * piece * 128;
            tma_load_3d_e(dst, &tmC, bar, pr * 128, y, blk);
            if (two) tma_load_3d_e(dst + CHUNK, &tmC, bar, pr * 128 + 64, y, blk);
          }
        }
        prefetch(j + p.stages);
      }
      if (!ok && lane == 0) {
        report_error(p.status, TW_ERR_MBAR_TIMEOUT);
        *abort_flag = 1;
      }
    }
  } else if (warp == 1) {
    // ---------------- MMA issuer ----------------
    // The whole warp walks through the loops and one elected lane issues: everything a descriptor is made of stays
    // uniform over the warp.
    if (n_tiles > 0) {
      const uint64_t desc_tile = make_smem_desc_sw128(smem_u32(smem), 16, 1024);          // K-major: scores
      const uint64_t desc_v = make_smem_desc_sw128(smem_u32(smem), CHUNK, 1024);          // MN-major: latent columns
      const uint64_t desc_q = make_smem_desc_sw128(smem_u32(s_q), 16, 1024);
      const uint64_t desc_p = make_smem_desc_sw128(smem_u32(s_p), 16, 1024);
      bool ok = mbar_wait_warp(q_ready, 0);
      auto issue_s = [&](int j) {
        const int st = j % p.stages;
        const uint32_t ph = (j / p.stages) & 1;
        const uint32_t tile_off = st * tile_bytes;
        const uint32_t d = tmem_base + (j & 1) * NC;
        for (int pr = 0; pr < pairs; ++pr) {
          if (!mbar_wait_warp(&full[st * LD_MAX_PAIRS + pr], ph)) return false;
          tc_fence_after_sync();
          // descriptors hold addresses in units of 16 bytes in their low bits: one addition each per instruction
          const uint64_t da = desc_tile + (tile_off + pr * 2 * CHUNK) / 16, db = desc_q + pr * (2 * NC * 128 / 16);
#pragma unroll
          for (int k = 0; k < 4; ++k) umma_ss_e(d, da + k * 2, db + k * 2, IDESC_S, (pr | k) != 0 ? 1u : 0u);
          if (2 * pr + 1 < p.chunks) {
#pragma unroll
            for (int k = 0; k < 4; ++k)
              umma_ss_e(d, da + CHUNK / 16 + k * 2, db + NC * 128 / 16 + k * 2, IDESC_S, 1u);
          }
          if (pr >= v_pairs) umma_commit_e(&empty[st * LD_MAX_PAIRS + pr]);     // no latent column in this pair
        }
        umma_commit_e(&s_full[j & 1]);
        return true;
      };
      auto tile_here = [&](int j) {
        const uint32_t ph = (j / p.stages) & 1;
        for (int pr = 0; pr < pairs; ++pr)
          if (!mbar_test_warp(&full[(j % p.stages) * LD_MAX_PAIRS + pr], ph)) return false;
        return true;
      };
      if (ok) ok = issue_s(0);
      for (int j = 0; ok && j < n_tiles; ++j) {
        // The next tile's score product goes first if its rows have landed before this tile's probabilities are there;
        // otherwise this tile's products go first, because they free the buffer that the load after the next waits for.
        bool ahead = j + 1 >= n_tiles;
        bool have_p = false;
        const uint64_t t_start = globaltimer_ns();
        while (!have_p) {
#pragma unroll 1
          for (int i = 0; i < 64 && !have_p; ++i) {
            if (!ahead && p.stages > 1 && tile_here(j + 1)) {
              ok = issue_s(j + 1);
              if (!ok) break;
              ahead = true;
            }
            have_p = ahead || p.stages == 1 ? mbar_try_wait_warp(p_ready, j & 1) : mbar_test_warp(p_ready, j & 1);
          }
          if (!ok || (!have_p && __any_sync(0xffffffffu, globaltimer_ns() - t_start > TW_WAIT_BUDGET_NS))) { ok = false; break; }
        }
        if (!ok) break;
        tc_fence_after_sync();
        const int st = j % p.stages;
        for (int m = 0; m < v_pairs; ++m) {
          const uint64_t da = desc_v + (st * tile_bytes + m * 2 * CHUNK) / 16;
          const uint32_t d = tmem_base + COL_O + m * NC;
#pragma unroll
          for (int k = 0; k < LD_BN / 16; ++k)
            umma_ss_e(d, da + k * (16 * 128 / 16), desc_p + ((k >> 2) * (NC * 128) + (k & 3) * 32) / 16, IDESC_O,
                    (j | k) != 0 ? 1u : 0u);
          if (EXACT) {
#pragma unroll
            for (int k = 0; k < LD_BN / 16; ++k)
              umma_ss_e(d, da + k * (16 * 128 / 16), desc_p + (P_LO + (k >> 2) * (NC * 128) + (k & 3) * 32) / 16, IDESC_O, 1u);
          }
          umma_commit_e(&empty[st * LD_MAX_PAIRS + m]);
        }
        umma_commit_e(o_done);
        if (!ahead) ok = issue_s(j + 1);
      }
      if (!ok && lane == 0) {
        report_error(p.status, TW_ERR_MBAR_TIMEOUT);
        *abort_flag = 1;
      }
    }
  } else {
    // ---------------- softmax + epilogue (warps 2..5) ----------------
    const int qr = warp & 3;                 // TMEM lane quarter this warp may touch
    const int r = qr * 32 + lane;            // key within the tile / latent column within a block in the epilogue
    const int sw = warp - 2;
    const int t = threadIdx.x - 64;          // 0..127
    const uint32_t t_lane = tmem_base + (static_cast<uint32_t>(qr * 32) << 16);

    float m_ref[NC], l_part[NC];
#pragma unroll
    for (int g = 0; g < NC; ++g) {
      m_ref[g] = -INFINITY;
      l_part[g] = 0.f;
    }
    bool ok = true;
    for (int j = 0; j < n_tiles; ++j) {
      // fixed trip count for all 128 threads: after a failed wait the remaining waits are skipped, not the iterations
      if (ok) ok = mbar_wait(&s_full[j & 1], (j >> 1) & 1);
      tc_fence_after_sync();
      uint32_t sv[NC];
      tmem_ld_cols(t_lane + (j & 1) * NC, sv);
      tmem_wait_ld();
      float* xm = xchg + (j & 1) * 4 * NC;
      const int key = (t_begin + j) * LD_BN + r;
      if (key >= kv_len || key < win_lo) {
#pragma unroll
        for (int g = 0; g < NC; ++g) sv[g] = __float_as_uint(-INFINITY);
      }
#pragma unroll
      for (int g4 = 0; g4 < NC; g4 += 4) {
        float4 mx;
        mx.x = warp_max_redux(__uint_as_float(sv[g4]));
        mx.y = warp_max_redux(__uint_as_float(sv[g4 + 1]));
        mx.z = warp_max_redux(__uint_as_float(sv[g4 + 2]));
        mx.w = warp_max_redux(__uint_as_float(sv[g4 + 3]));
        if (lane == 0) *reinterpret_cast<float4*>(xm + sw * NC + g4) = mx;
      }
      ld_softmax_sync();
      // a head's reference maximum moves when its maximum grew by more than 2^8 (rare after the first tiles); all 128
      // threads see the same maxima and decide alike
      float over = -1.f, mt[NC];
#pragma unroll
      for (int g4 = 0; g4 < NC; g4 += 4) {
        const float4 a = *reinterpret_cast<const float4*>(xm + g4);
        const float4 b = *reinterpret_cast<const float4*>(xm + NC + g4);
        const float4 c = *reinterpret_cast<const float4*>(xm + 2 * NC + g4);
        const float4 d = *reinterpret_cast<const float4*>(xm + 3 * NC + g4);
        mt[g4] = fmaxf(fmaxf(a.x, b.x), fmaxf(c.x, d.x)) * p.scale_log2;
        mt[g4 + 1] = fmaxf(fmaxf(a.y, b.y), fmaxf(c.y, d.y)) * p.scale_log2;
        mt[g4 + 2] = fmaxf(fmaxf(a.z, b.z), fmaxf(c.z, d.z)) * p.scale_log2;
        mt[g4 + 3] = fmaxf(fmaxf(a.w, b.w), fmaxf(c.w, d.w)) * p.scale_log2;
      }
      bool rescale = false;
      if (j == 0) {
#pragma unroll
        for (int g = 0; g < NC; ++g) m_ref[g] = mt[g];
      } else {
#pragma unroll
        for (int g = 0; g < NC; ++g) over = fmaxf(over, mt[g] - m_ref[g]);
        if (over > 8.f) {
          rescale = true;
#pragma unroll
          for (int g = 0; g < NC; ++g) {
            // mt becomes the factor of column g
            const float a = mt[g] > m_ref[g] + 8.f ? ld_exp2(m_ref[g] - mt[g]) : 1.f;
            if (mt[g] > m_ref[g] + 8.f) m_ref[g] = mt[g];
            l_part[g] *= a;
            mt[g] = a;
          }
        }
      }
      // P and O belong to the previous tile until its products are done. Every tile waits, needed or not: a parity
      // wait only tells that the phase before the current one has completed
      if (j > 0) {
        if (ok) ok = mbar_wait(o_done, (j - 1) & 1);
        tc_fence_after_sync();
      }
      uint8_t* p_buf = s_p + (r >> 6) * (NC * 128);
      const int kc = (r & 63) >> 3, ke = r & 7;
#pragma unroll
      for (int g = 0; g < NC; ++g) {
        const float pv = ld_exp2(fmaf(__uint_as_float(sv[g]), p.scale_log2, -m_ref[g]));
        l_part[g] += pv;
        uint8_t* at = p_buf + g * 128 + ((kc ^ (g & 7)) * 16) + ke * 2;
        const __nv_bfloat16 hi = __float2bfloat16(pv);
        *reinterpret_cast<__nv_bfloat16*>(at) = hi;
        if (EXACT) *reinterpret_cast<__nv_bfloat16*>(at + P_LO) = __float2bfloat16(pv - __bfloat162float(hi));
      }
      if (rescale) {
#pragma unroll 1
        for (int m = 0; m < v_pairs; ++m) {
          uint32_t ov[NC];
          tmem_ld_cols(t_lane + COL_O + m * NC, ov);
          tmem_wait_ld();
#pragma unroll
          for (int g = 0; g < NC; ++g) ov[g] = __float_as_uint(__uint_as_float(ov[g]) * mt[g]);
          tmem_st_cols(t_lane + COL_O + m * NC, ov);
        }
        tmem_wait_st();
      }
      tc_fence_before_sync();
      fence_proxy_async_smem();
      mbar_arrive(p_ready);       // arrive even after a failed wait so that the issuer is not left hanging
    }

    // row sums over the owners of the keys
    float* xs = xchg + (n_tiles & 1) * 4 * NC;
#pragma unroll
    for (int g = 0; g < NC; ++g) {
      const float l = warp_sum(l_part[g]);
      if (lane == 0) xs[sw * NC + g] = l;
    }
    ld_softmax_sync();
    if (n_tiles > 0 && ok) ok = mbar_wait(o_done, (n_tiles - 1) & 1);
    tc_fence_after_sync();
    if (p.splits == 1) {
      // O^T to [head][latent] through the tile buffers (nothing is in flight any more), then whole rows to memory
      __nv_bfloat16* s_o = reinterpret_cast<__nv_bfloat16*>(smem);
      const int ld_o = v_pairs * 128 + 8;
      float inv[NC];
#pragma unroll
      for (int g = 0; g < NC; ++g) {
        float l = (xs[g] + xs[NC + g]) + (xs[2 * NC + g] + xs[3 * NC + g]);
        if (p.sink != nullptr && g < G) l += ld_exp2(fmaf(p.sink[h0 + g], 1.4426950408889634f, -m_ref[g]));
        inv[g] = l > 0.f ? __fdividef(1.f, l) : 0.f;
      }
#pragma unroll 1
      for (int m = 0; m < v_pairs; ++m) {
        uint32_t ov[NC];
        tmem_ld_cols(t_lane + COL_O + m * NC, ov);
        tmem_wait_ld();
#pragma unroll
        for (int g = 0; g < NC; ++g)
          s_o[g * ld_o + m * 128 + r] = __float2bfloat16(n_tiles > 0 ? __uint_as_float(ov[g]) * inv[g] : 0.f);
      }
      ld_softmax_sync();
      if (ok) {
        const long long first = (static_cast<long long>(tok) * p.heads + h0) * p.kv_rank;
        if (p.kv_rank % 8 == 0) {
          const int per = p.kv_rank >> 3;
          for (int i = t; i < G * per; i += 128) {
            const int g = i / per, v = i - g * per;
            *reinterpret_cast<uint4*>(p.out + first + static_cast<long long>(i) * 8) =
                *reinterpret_cast<const uint4*>(s_o + g * ld_o + v * 8);
          }
        } else {
          for (int i = t; i < G * p.kv_rank; i += 128) {
            const int g = i / p.kv_rank;
            p.out[first + i] = s_o[g * ld_o + i - g * p.kv_rank];
          }
        }
      }
    } else if (ok) {
#pragma unroll 1
      for (int m = 0; m < v_pairs; ++m) {
        uint32_t ov[NC];
        tmem_ld_cols(t_lane + COL_O + m * NC, ov);
        tmem_wait_ld();
        const int d = m * 128 + r;
#pragma unroll
        for (int g = 0; g < NC; ++g) {
          if (g < G && d < p.kv_rank) {
            const long long pi = (static_cast<long long>(tok) * p.heads + h0 + g) * p.splits + split;
            p.part_o[pi * p.kv_rank + d] = n_tiles > 0 ? __uint_as_float(ov[g]) : 0.f;
            if (d == 0) {
              p.part_ml[pi * 2] = m_ref[g];
              p.part_ml[pi * 2 + 1] = (xs[g] + xs[NC + g]) + (xs[2 * NC + g] + xs[3 * NC + g]);
            }
          }
        }
      }
    }
    if (!ok) {
      report_error(p.status, TW_ERR_MBAR_TIMEOUT);
      *abort_flag = 1;
    }
  }

  if (*abort_flag) {
    // let copies and MMAs in flight land before shared memory and TMEM are given back
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after_sync();
    tmem_dealloc(tmem_base, TMEM_COLS);
  }
}

__global__ void __launch_bounds__(128)
latent_decode_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, int splits, int kv_rank,
                           const float* __restrict__ sink, int heads, __nv_bfloat16* __restrict__ out) {
  const long long item = blockIdx.x;
  float mm = -INFINITY, ll = 0.f;
  for (int s = 0; s < splits; ++s) mm = fmaxf(mm, part_ml[(item * splits + s) * 2]);
  if (sink != nullptr) ll = exp2f(fmaf(sink[item % heads], 1.4426950408889634f, -mm));
  for (int s = 0; s < splits; ++s) {
    const float m = part_ml[(item * splits + s) * 2];
    ll += m == -INFINITY ? 0.f : part_ml[(item * splits + s) * 2 + 1] * exp2f(m - mm);
  }
  const float inv = ll > 0.f ? 1.f / ll : 0.f;
  for (int d = threadIdx.x; d < kv_rank; d += blockDim.x) {
    float acc = 0.f;
    for (int s = 0; s < splits; ++s) {
      const float m = part_ml[(item * splits + s) * 2];
      if (m != -INFINITY) acc = fmaf(part_o[(item * splits + s) * kv_rank + d], exp2f(m - mm), acc);
    }
    out[item * kv_rank + d] = __float2bfloat16(acc * inv);
  }
}

template <int NC, bool EXACT>
static int launch_latent_decode(const void* cache, int num_blocks, LatentDecodeParams& p, int n, cudaStream_t stream) {
  CUtensorMap tm;
  {
    uint64_t dims[3] = {(uint64_t)p.row, (uint64_t)p.page, (uint64_t)num_blocks};
    uint64_t strides[2] = {(uint64_t)p.row * 2, (uint64_t)p.page * p.row * 2};
    uint32_t box[3] = {64, (uint32_t)(p.page < LD_BN ? p.page : LD_BN), 1};
    if (!make_tensor_map_bf16(&tm, cache, 3, dims, strides, box)) return 1;
  }
  CUtensorMap tmQ;
  {
    uint64_t dims[2] = {(uint64_t)p.row, (uint64_t)n * p.heads};
    uint64_t strides[1] = {(uint64_t)p.row * 2};
    uint32_t box[2] = {64, NC};
    if (!make_tensor_map_bf16(&tmQ, p.q, 2, dims, strides, box)) return 1;
  }
  const int tile_bytes = (p.chunks + 1) / 2 * 2 * LD_BN * 128, fixed = ld_fixed_bytes<NC, EXACT>(p.chunks);
  p.stages = (LD_SMEM_LIMIT - fixed) / tile_bytes;
  if (p.stages > LD_MAX_STAGES) p.stages = LD_MAX_STAGES;
  if (p.stages < 1) {
    set_last_error("latent_decode: rows of %d elements do not fit shared memory", p.row);
    return 1;
  }
  const int bytes = fixed + p.stages * tile_bytes;
  static thread_local int configured_dev = -1;
  int dev = 0;
  cudaGetDevice(&dev);
  if (configured_dev != dev) {
    const cudaError_t e =
        cudaFuncSetAttribute(latent_decode_kernel<NC, EXACT>, cudaFuncAttributeMaxDynamicSharedMemorySize, LD_SMEM_LIMIT);
    if (e != cudaSuccess) {
      set_last_error("latent_decode: cudaFuncSetAttribute failed: %s", cudaGetErrorString(e));
      return 1;
    }
    configured_dev = dev;
  }
  latent_decode_kernel<NC, EXACT><<<dim3(n, (p.heads + NC - 1) / NC, p.splits), LD_THREADS, bytes, stream>>>(tm, tmQ, p);
  cudaError_t e = cudaGetLastError();
  if (e == cudaSuccess && p.splits > 1) {
    latent_decode_merge_kernel<<<n * p.heads, 128, 0, stream>>>(p.part_o, p.part_ml, p.splits, p.kv_rank, p.sink,
                                                                 p.heads, p.out);
    e = cudaGetLastError();
  }
  if (e != cudaSuccess) {
    set_last_error("latent_decode launch failed: %s", cudaGetErrorString(e));
    return 1;
  }
  return 0;
}

}  // namespace tw

using namespace tw;

// qa [n, heads, row] absorbed queries, cache [num_blocks, page, row] (page a power of two, 8...128), out
// [n, heads, kv_rank]; part_o [n, heads, splits, kv_rank] and part_ml [n, heads, splits, 2] when splits > 1.
extern "C" int tw_latent_decode(const void* qa, const void* cache, int num_blocks, int page, const int* tok_seq,
                                const int* tok_kvlen, int n, const int* block_table, int max_blocks, void* out, int heads,
                                int row, int kv_rank, float scale, int window, const float* sink, int exact, int splits,
                                float* part_o, float* part_ml, uint32_t* status, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (row % 8 != 0 || row > 64 * 2 * LD_MAX_PAIRS || kv_rank > 512 || kv_rank > row || page < 8 || page > 128 || 128 % page != 0) {
    set_last_error("latent_decode: unsupported cache rows (row=%d, kv_rank=%d, page=%d)", row, kv_rank, page);
    return 1;
  }
  if (splits < 1) splits = 1;
  if (splits > 1 && (part_o == nullptr || part_ml == nullptr)) {
    set_last_error("latent_decode: splits need the partial-result workspace");
    return 1;
  }
  LatentDecodeParams p{reinterpret_cast<const __nv_bfloat16*>(qa), reinterpret_cast<__nv_bfloat16*>(out),
                       reinterpret_cast<const __nv_bfloat16*>(cache), tok_seq, tok_kvlen,
                       block_table, max_blocks, page, heads, row, kv_rank, splits, (row + 63) / 64, 1,
                       scale * 1.4426950408889634f, part_o, part_ml, status, window, sink};
  if (exact)
    return heads <= 16 ? launch_latent_decode<16, true>(cache, num_blocks, p, n, stream)
                       : launch_latent_decode<32, true>(cache, num_blocks, p, n, stream);
  return heads <= 16 ? launch_latent_decode<16, false>(cache, num_blocks, p, n, stream)
                     : launch_latent_decode<32, false>(cache, num_blocks, p, n, stream);
}
