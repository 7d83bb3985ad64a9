// Causal prefill attention in the expanded form of latent attention, for sm_100a: every head has keys of an unrotated
// part of its own and a rotated part shared by all heads, and values of another width. Keys and values of the context
// lie in contiguous workspaces (one matrix product from the gathered latents), not in pages.
//
// The kernel is the persistent form of attn_prefill_split.cu: a work item is one head of one 128-query tile, the item's
// key tiles are cut in two halves that two softmax groups process concurrently (own S, P, O in tensor memory, own K and
// V buffers in shared memory) and merge in the epilogue straight from tensor memory; P is the tensor-memory A operand
// of P V. What differs: a key tile is KC chunks of 64 columns, the first ones from the head's unrotated keys and the
// others from the shared rotated part (chunks are zero-filled behind each part's end by the tensor maps, so widths need
// not be multiples of 64); values are VC chunks; K and V have separate buffers because their sizes differ; the epilogue
// multiplies the output by sigmoid(gate), the output gate of the layer; and a sink per head may join the denominator.
//
// The windowed form (an instantiation of its own): an item visits the tiles that hold visible keys only, and the softmax
// weights reach the product with V as two bf16 terms, which keeps 16 bits of them (the leading terms in the upper half of
// the S columns, the others in the lower half); that product starts when the weights of a tile's first 64 keys are there.
//
// Roles (320 threads): warp 0 TMA producer, warp 1 MMA issuer, warps 2..5 softmax group A (one thread per query row),
// warps 6..9 group B. Every mbarrier wait is bounded; after a timeout the roles keep their trip counts, report
// TW_ERR_MBAR_TIMEOUT and leave through the tear-down.
#include "attn_prefill_common.cuh"
#include "tw_host.h"
#include "tw_kernels.h"
#include "tw_typed.cuh"

namespace tw {

constexpr int LP_MAX_SLOTS = 2;

template <int KC, int VC>
struct LatentPrefillSmem {
  static constexpr int K_BYTES = KC * ATT_HALF_BYTES;
  static constexpr int V_BYTES = VC * ATT_HALF_BYTES;
  static constexpr int LIMIT = 227 * 1024 - 256 - 1024 - K_BYTES;          // what K and V buffers of both groups may take
  static constexpr int KS = 2 * (2 * K_BYTES + V_BYTES) <= LIMIT ? 2 : 1;  // buffers per group
  static constexpr int VS = 2 * (KS * K_BYTES + 2 * V_BYTES) <= LIMIT ? 2 : 1;
  static constexpr int OFF_Q = 0;
  static constexpr int OFF_K = K_BYTES;                                    // [2 groups][KS]
  static constexpr int OFF_V = OFF_K + 2 * KS * K_BYTES;                   // [2 groups][VS]
  static constexpr int OFF_BAR = OFF_V + 2 * VS * V_BYTES;
  static constexpr int TOTAL = OFF_BAR + 256 + 1024;
  static_assert(2 * (KS * K_BYTES + VS * V_BYTES) <= LIMIT, "the tiles do not fit shared memory");
};

struct LatentPrefillParams {
  __nv_bfloat16* out; long long ldo;
  const __nv_bfloat16* gate; long long ldg;     // null: no output gate
  const int *cu_q, *kv_lens, *tile_seq, *tile_q0;
  const int* ctx_begin;                         // [B] workspace row of a sequence's key 0 (may lie before the first row
                                                // when a window leaves the first keys out)
  int heads, dim, vdim, k_chunks;               // k_chunks: chunks of the unrotated part
  float scale_log2;
  uint32_t* status;
  int window;                                   // > 0: a query sees the last `window` keys, itself among them
  const float* sink;                            // [heads] or null: exp(sink) joins the denominator
};

struct LatentPrefillItem {
  int head, q_begin, q0, rows_valid, pos0, ctx, j_lo, n_tiles, n_a;
};

template <bool WINDOW>
__device__ __forceinline__ LatentPrefillItem latent_item(const LatentPrefillParams& p, int idx) {
  LatentPrefillItem it;
  const int tile = idx / p.heads;
  it.head = idx - tile * p.heads;
  const int seq = p.tile_seq[tile];
  it.q0 = p.tile_q0[tile];
  it.q_begin = p.cu_q[seq];
  const int q_len = p.cu_q[seq + 1] - it.q_begin;
  const int kv_len = p.kv_lens[seq];
  it.ctx = p.ctx_begin[seq];
  it.rows_valid = min(ATT_BM, q_len - it.q0);
  it.pos0 = kv_len - q_len + it.q0;
  it.j_lo = WINDOW ? max(0, it.pos0 - p.window + 1) / ATT_BN : 0;
  it.n_tiles = (min(kv_len, it.pos0 + it.rows_valid) + ATT_BN - 1) / ATT_BN - it.j_lo;
  it.n_a = (it.n_tiles + 1) / 2;
  return it;
}

template <int KC, int VC, bool WINDOW>
__global__ void __launch_bounds__(ATT_THREADS, 1)
latent_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                      const __grid_constant__ CUtensorMap tmR, const __grid_constant__ CUtensorMap tmV,
                      const LatentPrefillParams p, const int total_items) {
  using S = LatentPrefillSmem<KC, VC>;
  constexpr int DV = VC * 64;
  constexpr uint32_t IDESC_QK = make_idesc_bf16(ATT_BM, ATT_BN, 0, 0);
  constexpr uint32_t IDESC_PV = make_idesc_bf16(ATT_BM, DV, 0, 1);
  constexpr uint32_t TMEM_COLS = 512;
  constexpr uint32_t COL_S = 0;     // S_A at 0, S_B at 128; P_g lives in columns [64, 128) of S_g
  constexpr uint32_t COL_P = 64;
  constexpr uint32_t COL_O = 256;   // O_A at 256, O_B at 384

  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) &
                                             ~static_cast<uintptr_t>(1023));
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + S::OFF_BAR);
  uint64_t* q_full = bars + 0;
  uint64_t* q_empty = bars + 1;
  uint64_t* k_full = bars + 2;        // [2][LP_MAX_SLOTS]
  uint64_t* k_empty = bars + 6;
  uint64_t* v_full = bars + 10;
  uint64_t* v_empty = bars + 14;
  uint64_t* s_full = bars + 18;       // [2]
  uint64_t* p_ready = bars + 20;      // [2]
  uint64_t* o_done = bars + 22;       // [2]
  uint64_t* epi_done = bars + 24;
  uint64_t* p_half = bars + 25;       // [2], windowed form: weights of the first 64 keys
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 27);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5;
  const int lane = threadIdx.x & 31;
  const int G = gridDim.x;
  const int cta = blockIdx.x;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    mbar_init(q_empty, 1);
    for (int i = 0; i < 2 * LP_MAX_SLOTS; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&v_empty[i], 1);
    }
    for (int g = 0; g < 2; ++g) {
      mbar_init(&s_full[g], 1);
      mbar_init(&p_ready[g], 128);
      mbar_init(&p_half[g], 128);
      mbar_init(&o_done[g], 1);
    }
    mbar_init(epi_done, ATT_SOFTMAX_THREADS);
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
    // ---------------- TMA producer ----------------
    if (lane == 0) {
      tma_prefetch_desc(&tmQ);
      tma_prefetch_desc(&tmK);
      tma_prefetch_desc(&tmR);
      tma_prefetch_desc(&tmV);
      uint32_t ek[2] = {0u, 0u}, ev[2] = {0u, 0u};      // K and V tiles loaded so far, per group
      bool ok = true;
      int items_done = 0;
      for (int round = 0; ok; ++round) {
        const int idx = split_item_index(round, cta, G);
        if (idx >= total_items) break;
        const LatentPrefillItem it = latent_item<WINDOW>(p, idx);
        if (items_done > 0 && !mbar_wait(q_empty, (items_done - 1) & 1)) { ok = false; break; }
        mbar_expect_tx(q_full, S::K_BYTES);
#pragma unroll
        for (int c = 0; c < KC; ++c)
          tma_load_3d(smem + S::OFF_Q + c * ATT_HALF_BYTES, &tmQ, q_full,
                      c < p.k_chunks ? c * 64 : p.dim + (c - p.k_chunks) * 64, it.head, it.q_begin + it.q0);
        auto load_k = [&](int g, int j) {
          const int slot = ek[g] % S::KS;
          if (!mbar_wait(&k_empty[g * LP_MAX_SLOTS + slot], ((ek[g] / S::KS) & 1) ^ 1)) return false;
          uint64_t* bar = &k_full[g * LP_MAX_SLOTS + slot];
          mbar_expect_tx(bar, S::K_BYTES);
          uint8_t* dst = smem + S::OFF_K + (g * S::KS + slot) * S::K_BYTES;
#pragma unroll
          for (int c = 0; c < KC; ++c) {
            if (c < p.k_chunks) tma_load_3d(dst + c * ATT_HALF_BYTES, &tmK, bar, c * 64, it.head, it.ctx + j * ATT_BN);
            else tma_load_2d(dst + c * ATT_HALF_BYTES, &tmR, bar, (c - p.k_chunks) * 64, it.ctx + j * ATT_BN);
          }
          ++ek[g];
          return true;
        };
        auto load_v = [&](int g, int j) {
          const int slot = ev[g] % S::VS;
          if (!mbar_wait(&v_empty[g * LP_MAX_SLOTS + slot], ((ev[g] / S::VS) & 1) ^ 1)) return false;
          uint64_t* bar = &v_full[g * LP_MAX_SLOTS + slot];
          mbar_expect_tx(bar, S::V_BYTES);
          uint8_t* dst = smem + S::OFF_V + (g * S::VS + slot) * S::V_BYTES;
#pragma unroll
          for (int c = 0; c < VC; ++c)
            tma_load_3d(dst + c * ATT_HALF_BYTES, &tmV, bar, c * 64, it.head, it.ctx + j * ATT_BN);
          ++ev[g];
          return true;
        };
        const int n_b = it.n_tiles - it.n_a;
        for (int t = 0; t < it.n_a && ok; ++t) {
          ok = load_k(0, it.j_lo + t);
          if (ok && t < n_b) ok = load_k(1, it.j_lo + it.n_a + t);
          if (ok) ok = load_v(0, it.j_lo + t);
          if (ok && t < n_b) ok = load_v(1, it.j_lo + it.n_a + t);
        }
        ++items_done;
      }
      if (!ok) {
        report_error(p.status, TW_ERR_MBAR_TIMEOUT);
        *abort_flag = 1;
      }
    }
  } else if (warp == 1) {
    // ---------------- MMA issuer ----------------
    if (lane == 0) {
      uint32_t ek[2] = {0u, 0u};          // key tiles whose scores have been issued, per group
      uint32_t cnt[2] = {0u, 0u};         // key tiles whose P V has been issued, per group
      const uint32_t q_addr = smem_u32(smem + S::OFF_Q);
      bool ok = true;
      int items_done = 0;
      for (int round = 0; ok; ++round) {
        const int idx = split_item_index(round, cta, G);
        if (idx >= total_items) break;
        const LatentPrefillItem it = latent_item<WINDOW>(p, idx);
        const int n_b = it.n_tiles - it.n_a;
        if (!mbar_wait(q_full, items_done & 1)) { ok = false; break; }
        // S_g carried the (m, l) exchange of the previous item's epilogue
        if (items_done > 0 && !mbar_wait(epi_done, (items_done - 1) & 1)) { ok = false; break; }
        tc_fence_after_sync();
        int qk_issued = 0;
        auto issue_qk = [&](int g) {
          const int slot = ek[g] % S::KS;
          if (!mbar_wait(&k_full[g * LP_MAX_SLOTS + slot], (ek[g] / S::KS) & 1)) return false;
          tc_fence_after_sync();
          const uint32_t k_addr = smem_u32(smem + S::OFF_K + (g * S::KS + slot) * S::K_BYTES);
#pragma unroll
          for (int k = 0; k < KC * 4; ++k) {
            const uint32_t off = (k >> 2) * ATT_HALF_BYTES + (k & 3) * 32;
            umma_ss(tmem_base + COL_S + g * 128, make_smem_desc_sw128(q_addr + off, 16, 1024),
                    make_smem_desc_sw128(k_addr + off, 16, 1024), IDESC_QK, k != 0 ? 1u : 0u);
          }
          umma_commit(&k_empty[g * LP_MAX_SLOTS + slot]);
          umma_commit(&s_full[g]);
          ++ek[g];
          if (++qk_issued == it.n_tiles) umma_commit(q_empty);   // the Q tile may be replaced once these are done
          return true;
        };
        auto issue_pv = [&](int g, bool first) {
          if (!mbar_wait(WINDOW ? &p_half[g] : &p_ready[g], cnt[g] & 1)) return false;
          const int slot = cnt[g] % S::VS;
          if (!mbar_wait(&v_full[g * LP_MAX_SLOTS + slot], (cnt[g] / S::VS) & 1)) return false;
          tc_fence_after_sync();
          const uint32_t v_addr = smem_u32(smem + S::OFF_V + (g * S::VS + slot) * S::V_BYTES);
          auto pv = [&](int k, uint32_t col, bool init) {
            umma_ts(tmem_base + COL_O + g * 128, tmem_base + COL_S + g * 128 + col + k * 8,
                    make_smem_desc_sw128(v_addr + k * 16 * 128, ATT_HALF_BYTES, 1024), IDESC_PV, init ? 0u : 1u);
          };
#pragma unroll
          for (int k = 0; k < ATT_BN / 16; ++k) {
            if (WINDOW && k == 4) {
              if (!mbar_wait(&p_ready[g], cnt[g] & 1)) return false;
              tc_fence_after_sync();
            }
            pv(k, COL_P, first && k == 0);
            if (WINDOW) pv(k, 0, false);
          }
          umma_commit(&v_empty[g * LP_MAX_SLOTS + slot]);
          umma_commit(&o_done[g]);
          ++cnt[g];
          return true;
        };
        ok = issue_qk(0);
        if (ok && n_b > 0) ok = issue_qk(1);
        for (int t = 0; ok && t < it.n_a; ++t) {
          ok = issue_pv(0, t == 0);
          if (ok && t + 1 < it.n_a) ok = issue_qk(0);
          if (ok && t < n_b) ok = issue_pv(1, t == 0);
          if (ok && t + 1 < n_b) ok = issue_qk(1);
        }
        ++items_done;
      }
      if (!ok) {
        report_error(p.status, TW_ERR_MBAR_TIMEOUT);
        *abort_flag = 1;
      }
    }
  } else {
    // ---------------- softmax + epilogue: warps 2..5 group A, warps 6..9 group B ----------------
    const int g = (warp - 2) >> 2;
    const int qr = warp & 3;                        // TMEM lane quarter of this warp
    const int r = qr * 32 + lane;                   // row within the tile
    const uint32_t t_lane = tmem_base + (static_cast<uint32_t>(qr * 32) << 16);
    const uint32_t t_s = t_lane + COL_S + g * 128;
    const uint32_t t_p = t_s + COL_P;
    uint32_t cnt = 0;                               // key tiles this group has processed
    bool ok = true;
    for (int round = 0;; ++round) {
      const int idx = split_item_index(round, cta, G);
      if (idx >= total_items) break;
      const LatentPrefillItem it = latent_item<WINDOW>(p, idx);
      const int n_b = it.n_tiles - it.n_a;
      const int n_mine = g == 0 ? it.n_a : n_b;
      const int j0 = it.j_lo + (g == 0 ? 0 : it.n_a);
      const int pos = it.pos0 + min(r, it.rows_valid - 1);   // padding rows copy the last valid row's mask
      const int pos_w = WINDOW ? pos - p.window + 1 : 0;     // first key this row sees
      float m_ref = -INFINITY;   // softmax reference (a stale running maximum), log2 domain
      float l_sum = 0.f;
      for (int t = 0; t < n_mine; ++t) {
        if (ok) ok = mbar_wait(&s_full[g], cnt & 1);
        tc_fence_after_sync();
        const int k_base = (j0 + t) * ATT_BN;
        // warp-uniform: lane 0 holds the warp's smallest position, lane 31 its largest
        bool need_mask = (k_base + ATT_BN - 1) > __shfl_sync(0xffffffffu, pos, 0);
        if (WINDOW) need_mask = need_mask || k_base < __shfl_sync(0xffffffffu, pos_w, 31);
        // The row's 128 scores come to registers in one go (four loads in flight, one wait): the latency of
        // tensor-memory loads is paid once per tile, and everything below runs from registers.
        uint32_t s0[32], s1[32], s2[32], s3[32];
        tmem_ld_32x32(t_s, s0);
        tmem_ld_32x32(t_s + 32, s1);
        tmem_ld_32x32(t_s + 64, s2);
        tmem_ld_32x32(t_s + 96, s3);
        tmem_wait_ld();
        if (need_mask) {
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            auto hidden = [&](int k) { return k > pos || (WINDOW && k < pos_w); };
            if (hidden(k_base + i)) s0[i] = __float_as_uint(-INFINITY);
            if (hidden(k_base + 32 + i)) s1[i] = __float_as_uint(-INFINITY);
            if (hidden(k_base + 64 + i)) s2[i] = __float_as_uint(-INFINITY);
            if (hidden(k_base + 96 + i)) s3[i] = __float_as_uint(-INFINITY);
          }
        }
        // row maximum: three-input max, one chain per chunk
        float m4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          m4[0] = max3f(m4[0], __uint_as_float(s0[2 * i]), __uint_as_float(s0[2 * i + 1]));
          m4[1] = max3f(m4[1], __uint_as_float(s1[2 * i]), __uint_as_float(s1[2 * i + 1]));
          m4[2] = max3f(m4[2], __uint_as_float(s2[2 * i]), __uint_as_float(s2[2 * i + 1]));
          m4[3] = max3f(m4[3], __uint_as_float(s3[2 * i]), __uint_as_float(s3[2 * i + 1]));
        }
        const float mx = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3])) * p.scale_log2;
        float alpha = 1.f;
        bool rescale = false;
        if (t == 0) {
          m_ref = mx;
        } else if (mx > m_ref + 8.f) {
          alpha = fast_exp2(m_ref - mx);
          m_ref = mx;
          rescale = true;
        }
        // a row of group B can have every key of its first tiles masked: its reference stays -inf and the
        // exponentials below must see a finite subtrahend
        const float m_use = (m_ref == -INFINITY) ? 0.f : m_ref;
        // exponentials, two scores per instruction where the ISA has a packed form (scale and subtract,
        // running sum, bf16 conversion); 32 keys become 16 columns of P, which overwrites S columns
        // 64..127 (every score is in registers by now)
        const float2 sc2 = make_float2(p.scale_log2, p.scale_log2);
        const float2 nm2 = make_float2(-m_use, -m_use);
        float2 sum2[2] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
        uint32_t pk[16], lo[16];
        auto exp_chunk = [&](const uint32_t (&buf)[32]) {
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            const float2 x = fma2(make_float2(__uint_as_float(buf[2 * i]), __uint_as_float(buf[2 * i + 1])), sc2, nm2);
            const float2 e = make_float2(fast_exp2(x.x), fast_exp2(x.y));
            sum2[i & 1] = fadd2(sum2[i & 1], e);
            if (WINDOW) split_weights(e, pk[i], lo[i]);
            else pk[i] = pack_bf16x2(e.x, e.y);
          }
        };
        auto store_chunk = [&](int chunk) {
          tmem_st_32x16(t_p + chunk * 16, pk);
          if (WINDOW) tmem_st_32x16(t_s + chunk * 16, lo);
        };
        exp_chunk(s0);
        store_chunk(0);
        exp_chunk(s1);
        store_chunk(1);
        if (t > 0 && __any_sync(0xffffffffu, rescale)) {
          // O_g may be touched once P V of the previous tile has completed
          if (ok) ok = mbar_wait(&o_done[g], (cnt - 1) & 1);
          tc_fence_after_sync();
          const uint32_t t_o = t_lane + COL_O + g * 128;
#pragma unroll 1
          for (int c = 0; c < DV / 32; ++c) {
            uint32_t v[32];
            tmem_ld_32x32(t_o + c * 32, v);
            tmem_wait_ld();
#pragma unroll
            for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * alpha);
            tmem_st_32x32(t_o + c * 32, v);
          }
        }
        if (WINDOW) {
          tmem_wait_st();
          tc_fence_before_sync();
          mbar_arrive(&p_half[g]);      // (O_g is scaled by then: the product may go on)
        }
        exp_chunk(s2);
        store_chunk(2);
        exp_chunk(s3);
        store_chunk(3);
        l_sum = l_sum * alpha + ((sum2[0].x + sum2[0].y) + (sum2[1].x + sum2[1].y));
        tmem_wait_st();
        tc_fence_before_sync();
        mbar_arrive(&p_ready[g]);   // arrive even after a failed wait so the issuer is not left waiting
        ++cnt;
      }
      if (n_mine > 0 && ok) ok = mbar_wait(&o_done[g], (cnt - 1) & 1);
      tc_fence_after_sync();
      // ---- epilogue: merge the two halves of the key range; group g writes output columns [g DV/2, (g+1) DV/2) ----
      tmem_st_32x2(t_s, __float_as_uint(m_ref), __float_as_uint(l_sum));
      tmem_wait_st();
      tc_fence_before_sync();
      split_pair_sync(qr);
      tc_fence_after_sync();
      uint32_t om_u, ol_u;
      tmem_ld_32x2(t_lane + COL_S + (g ^ 1) * 128, om_u, ol_u);
      tmem_wait_ld();
      tc_fence_before_sync();
      mbar_arrive(epi_done);        // S_A and S_B are free for the next item
      const float o_m = __uint_as_float(om_u), o_l = __uint_as_float(ol_u);
      const float m_all = fmaxf(m_ref, o_m);
      const float f_me = fast_exp2(m_ref - m_all), f_ot = fast_exp2(o_m - m_all);
      float l_all = l_sum * f_me + o_l * f_ot;
      if (p.sink != nullptr) l_all += fast_exp2(fmaf(p.sink[it.head], 1.4426950408889634f, -m_all));
      const float inv = 1.f / l_all;
      const float f_a = (g == 0 ? f_me : f_ot) * inv, f_b = (g == 0 ? f_ot : f_me) * inv;
      const long long out_row = it.q_begin + it.q0 + r;
      __nv_bfloat16* orow = p.out + out_row * p.ldo + it.head * p.vdim;
      const __nv_bfloat16* grow = p.gate != nullptr ? p.gate + out_row * p.ldg + it.head * p.vdim : nullptr;
#pragma unroll 1
      for (int c = 0; c < DV / 64; ++c) {
        uint32_t a[32], b[32];
        const int col0 = g * (DV / 2) + c * 32;
        tmem_ld_32x32(t_lane + COL_O + col0, a);
        if (n_b > 0) tmem_ld_32x32(t_lane + COL_O + col0 + 128, b);
        tmem_wait_ld();
        if (n_b > 0) {
#pragma unroll
          for (int i = 0; i < 32; ++i)
            a[i] = __float_as_uint(__uint_as_float(a[i]) * f_a + __uint_as_float(b[i]) * f_b);
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i) a[i] = __float_as_uint(__uint_as_float(a[i]) * f_a);
        }
        if (r < it.rows_valid && ok) {
#pragma unroll
          for (int q8 = 0; q8 < 4; ++q8) {
            if (col0 + q8 * 8 < p.vdim) {
              float v[8];
#pragma unroll
              for (int i = 0; i < 8; ++i) v[i] = __uint_as_float(a[8 * q8 + i]);
              if (grow != nullptr) {
                float s[8];
                ld8(grow + col0 + q8 * 8, s);
#pragma unroll
                for (int i = 0; i < 8; ++i) v[i] *= sigmoid_t<__nv_bfloat16>(s[i]);
              }
              st8(orow + col0 + q8 * 8, v);
            }
          }
        }
      }
      // both groups have read O_A and O_B before either signals the first P of the next item
      tc_fence_before_sync();
      split_pair_sync(qr);
      tc_fence_after_sync();
    }
    if (!ok) {
      report_error(p.status, TW_ERR_MBAR_TIMEOUT);
      *abort_flag = 1;
    }
  }

  // ---------------- tear-down ----------------
  if (*abort_flag) {
    // give copies that may still be in flight time to land before shared memory is released
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

template <int KC, int VC, bool WINDOW>
static int launch_latent_prefill(const CUtensorMap& tmQ, const CUtensorMap& tmK, const CUtensorMap& tmR,
                                 const CUtensorMap& tmV, const LatentPrefillParams& p, int num_tiles,
                                 cudaStream_t stream) {
  using S = LatentPrefillSmem<KC, VC>;
  auto kern = latent_prefill_kernel<KC, VC, WINDOW>;
  static thread_local int configured_dev = -1;
  int dev = 0;
  cudaGetDevice(&dev);
  if (configured_dev != dev) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, S::TOTAL);
    if (e != cudaSuccess) {
      set_last_error("latent_prefill: cudaFuncSetAttribute(smem=%d) failed: %s", S::TOTAL, cudaGetErrorString(e));
      return 1;
    }
    configured_dev = dev;
  }
  const long long items = static_cast<long long>(num_tiles) * p.heads;
  int grid = device_sm_count();
  if (items < grid) grid = static_cast<int>(items);
  kern<<<grid, ATT_THREADS, S::TOTAL, stream>>>(tmQ, tmK, tmR, tmV, p, static_cast<int>(items));
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) {
    set_last_error("latent_prefill launch failed: %s", cudaGetErrorString(e));
    return 1;
  }
  return 0;
}

}  // namespace tw

using namespace tw;

// q [T, heads * (dim + rot)] with the rotated tails, kv [ctx_rows, heads * dim | heads * vdim] (row stride ldkv),
// kr [ctx_rows, rot] (row stride ldr); key k of sequence b is workspace row ctx_begin[b] + k, for every key from the first
// visible one's tile of 128 on.
extern "C" int tw_latent_prefill(const void* q, long long ldq, int T, const void* kv, long long ldkv, const void* kr,
                                 long long ldr, int ctx_rows, const int* ctx_begin, void* out, long long ldo,
                                 const void* gate, long long ldg, const int* cu_q, const int* kv_lens,
                                 const int* tile_seq, const int* tile_q0, int num_tiles, int heads, int dim, int rot,
                                 int vdim, float scale, int window, const float* sink, uint32_t* status,
                                 cudaStream_t stream) {
  if (num_tiles <= 0) return 0;
  const int kc = (dim + 63) / 64 + (rot + 63) / 64, vc = (vdim + 63) / 64;
  if (dim % 8 != 0 || rot % 8 != 0 || vdim % 8 != 0 || ldq % 8 != 0 || ldkv % 8 != 0 || ldr % 8 != 0 || ldo % 8 != 0 ||
      ldg % 8 != 0 || kc < 2 || vc < 1 || kc + vc > 5 || vc > 2) {
    set_last_error("latent_prefill: unsupported head sizes (dim=%d, rot=%d, vdim=%d)", dim, rot, vdim);
    return 1;
  }
  CUtensorMap tmQ, tmK, tmR, tmV;
  {
    uint64_t dims[3] = {(uint64_t)(dim + rot), (uint64_t)heads, (uint64_t)T};
    uint64_t strides[2] = {(uint64_t)(dim + rot) * 2, (uint64_t)ldq * 2};
    uint32_t box[3] = {64, 1, ATT_BM};
    if (!make_tensor_map_bf16(&tmQ, q, 3, dims, strides, box)) return 1;
  }
  {
    uint64_t dims[3] = {(uint64_t)dim, (uint64_t)heads, (uint64_t)ctx_rows};
    uint64_t strides[2] = {(uint64_t)dim * 2, (uint64_t)ldkv * 2};
    uint32_t box[3] = {64, 1, ATT_BN};
    if (!make_tensor_map_bf16(&tmK, kv, 3, dims, strides, box)) return 1;
    dims[0] = (uint64_t)vdim;
    strides[0] = (uint64_t)vdim * 2;
    if (!make_tensor_map_bf16(&tmV, reinterpret_cast<const __nv_bfloat16*>(kv) + static_cast<long long>(heads) * dim, 3,
                              dims, strides, box))
      return 1;
  }
  {
    uint64_t dims[2] = {(uint64_t)rot, (uint64_t)ctx_rows};
    uint64_t strides[1] = {(uint64_t)ldr * 2};
    uint32_t box[2] = {64, ATT_BN};
    if (!make_tensor_map_bf16(&tmR, kr, 2, dims, strides, box)) return 1;
  }
  using bf = __nv_bfloat16;
  const LatentPrefillParams p{reinterpret_cast<bf*>(out), ldo, reinterpret_cast<const bf*>(gate), ldg, cu_q, kv_lens,
                              tile_seq, tile_q0, ctx_begin, heads, dim, vdim, (dim + 63) / 64,
                              scale * 1.4426950408889634f, status, window, sink};
#define TW_CASE(K, V) \
  if (kc == K && vc == V)                                                                               \
    return window > 0 ? launch_latent_prefill<K, V, true>(tmQ, tmK, tmR, tmV, p, num_tiles, stream)      \
                      : launch_latent_prefill<K, V, false>(tmQ, tmK, tmR, tmV, p, num_tiles, stream);
  TW_CASE(2, 1) TW_CASE(2, 2) TW_CASE(3, 1) TW_CASE(3, 2) TW_CASE(4, 1)
#undef TW_CASE
  set_last_error("latent_prefill: unsupported head sizes (dim=%d, rot=%d, vdim=%d)", dim, rot, vdim);
  return 1;
}
