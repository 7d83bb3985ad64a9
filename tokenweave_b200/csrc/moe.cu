// Mixture-of-experts routing kernels.
//
//   tw_moe_router      (Mixtral: 8 experts, top-2, softmax then renormalise) gate GEMV (x . Wg^T, fp32) + softmax + top-k + renormalise, one kernel.
//                      Reference: replicated gate linear, then csrc/moe/topk_softmax_kernels.cu
//                      and the renormalisation in fused_moe.py:831-844.
//   tw_moe_route       the general router, any number of experts up to 256, bf16 and fp32: scores are the softmax over all
//                      experts or the sigmoid of each logit, the top ones are chosen by score + correction, their weights
//                      are the scores, or those over their sum; further rows of the same matrix give sigmoid gates (of a
//                      shared expert)
//   tw_moe_align       counting sort of (token, k) pairs by expert with every expert's segment
//                      padded to the GEMM's 128-row tile; emits the expert of each row tile, the
//                      number of tiles, the sorted position of every pair.
//                      Reference: csrc/moe/moe_align_sum_kernels.cu:24-112.
//   tw_moe_scatter     copies token rows into expert-sorted order (the A operand of the grouped
//                      GEMM) and the routing weight of each sorted row.
//   tw_moe_combine     out[t] = sum_k y_sorted[pos[t,k]] (+ gate[t] * shared[t], or + shared[t]) (weights were applied by
//                      a grouped GEMM's epilogue). Reference: moe_sum_kernel,
//                      moe_align_sum_kernels.cu:277-293.
#include "tw_common.cuh"
#include "tw_host.h"
#include "tw_kernels.h"
#include "tw_mma.cuh"
#include "tw_typed.cuh"

namespace tw {

constexpr int MOE_MAX_EXPERTS = 256;
constexpr int MOE_MAX_TOPK = 8;

__device__ __forceinline__ float2 moe_ffma2(float2 a, float2 b, float2 c) {
  uint64_t ra, rb, rc, rd;
  asm("mov.b64 %0, {%1, %2};" : "=l"(ra) : "f"(a.x), "f"(a.y));
  asm("mov.b64 %0, {%1, %2};" : "=l"(rb) : "f"(b.x), "f"(b.y));
  asm("mov.b64 %0, {%1, %2};" : "=l"(rc) : "f"(c.x), "f"(c.y));
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(rd) : "l"(ra), "l"(rb), "l"(rc));
  float2 d;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(d.x), "=f"(d.y) : "l"(rd));
  return d;
}

// TPW tokens per warp, persistent CTAs. The gate weight [E, H] lives in shared memory; a warp reads (and converts)
// every 16 bytes of it once for its TPW tokens, and the multiply-adds are the packed two-wide fp32 form of sm_100:
// this is about one instruction per multiply-add where one token per warp with scalar FMAs took 2.1.
template <int E, int TPW>
__global__ void __launch_bounds__(512)       // 16 warps per SM: 128 registers each for the TPW x E accumulators
moe_router_kernel(const __nv_bfloat16* __restrict__ x, long long ldx,
                  const __nv_bfloat16* __restrict__ wg, float* __restrict__ topk_w,
                  int* __restrict__ topk_ids, float* __restrict__ logits_out, int T, int H, int topk,
                  int renormalize) {
  extern __shared__ uint8_t smem_raw[];
  uint4* wsm = reinterpret_cast<uint4*>(smem_raw);
  const int nvec = H >> 3;
  for (int i = threadIdx.x; i < E * nvec; i += blockDim.x)
    wsm[i] = reinterpret_cast<const uint4*>(wg)[i];
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, wpb = blockDim.x >> 5;
  for (int tb = (blockIdx.x * wpb + warp) * TPW; tb < T; tb += gridDim.x * wpb * TPW) {
    float2 acc[TPW][E];            // .x: even elements of the row, .y: odd ones
#pragma unroll
    for (int i = 0; i < TPW; ++i)
#pragma unroll
      for (int e = 0; e < E; ++e) acc[i][e] = make_float2(0.f, 0.f);
    const uint4* xr[TPW];
#pragma unroll
    for (int i = 0; i < TPW; ++i)          // tokens past the end re-read the last row; their results are dropped
      xr[i] = reinterpret_cast<const uint4*>(x + static_cast<long long>(min(tb + i, T - 1)) * ldx);
    // the row pieces of the NEXT step are requested before this step's arithmetic: with 16 warps per SM the loads
    // of one step alone would leave the memory system idle while the warps multiply
    uint4 xv[TPW];
#pragma unroll
    for (int i = 0; i < TPW; ++i) xv[i] = lane < nvec ? xr[i][lane] : make_uint4(0u, 0u, 0u, 0u);
    for (int v = lane; v < nvec; v += 32) {
      float2 xf[TPW][4];
#pragma unroll
      for (int i = 0; i < TPW; ++i) {
        const uint32_t* xu = reinterpret_cast<const uint32_t*>(&xv[i]);
#pragma unroll
        for (int j = 0; j < 4; ++j) xf[i][j] = unpack_bf16x2(xu[j]);
      }
      if (v + 32 < nvec) {
#pragma unroll
        for (int i = 0; i < TPW; ++i) xv[i] = xr[i][v + 32];
      }
#pragma unroll
      for (int e = 0; e < E; ++e) {
        const uint4 wv = wsm[e * nvec + v];
        const uint32_t* wu = reinterpret_cast<const uint32_t*>(&wv);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float2 wf = unpack_bf16x2(wu[j]);
#pragma unroll
          for (int i = 0; i < TPW; ++i) acc[i][e] = moe_ffma2(xf[i][j], wf, acc[i][e]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < TPW; ++i) {
      float logit[E];
#pragma unroll
      for (int e = 0; e < E; ++e) logit[e] = warp_sum(acc[i][e].x + acc[i][e].y);
      const int t = tb + i;
      if (lane == i && t < T) {             // one lane per token: the TPW tails run side by side
        float mx = logit[0];
#pragma unroll
        for (int e = 1; e < E; ++e) mx = fmaxf(mx, logit[e]);
        float p[E];
        float den = 0.f;
#pragma unroll
        for (int e = 0; e < E; ++e) {
          p[e] = __expf(logit[e] - mx);
          den += p[e];
        }
        if (logits_out != nullptr) {
#pragma unroll
          for (int e = 0; e < E; ++e) logits_out[static_cast<long long>(t) * E + e] = logit[e];
        }
        float wsum = 0.f;
        float sel_w[MOE_MAX_TOPK];
        int sel_i[MOE_MAX_TOPK];
        for (int k = 0; k < topk; ++k) {
          int bi = 0;
          float bv = -1.f;
#pragma unroll
          for (int e = 0; e < E; ++e) {
            if (p[e] > bv) { bv = p[e]; bi = e; }
          }
          sel_w[k] = bv / den;
          sel_i[k] = bi;
          wsum += sel_w[k];
#pragma unroll
          for (int e = 0; e < E; ++e)
            if (e == bi) p[e] = -2.f;
        }
        for (int k = 0; k < topk; ++k) {
          topk_w[static_cast<long long>(t) * topk + k] = renormalize ? sel_w[k] / wsum : sel_w[k];
          topk_ids[static_cast<long long>(t) * topk + k] = sel_i[k];
        }
      }
    }
  }
}

// ---- general router --------------------------------------------------------------------------------------------
constexpr int ROUTE_MAX_TOPK = 32, ROUTE_MAX_GATES = 8;

struct RouteArgs {
  const void* x; long long ldx;
  const void* w; long long ldw;             // [E + gates, H]
  const float* correction;                  // [E] or null
  float* topk_w; int* topk_ids;             // [T, topk]
  float* gate;                              // [T, gates]
  int T, H, E, gates, topk;
  int sigmoid, normalize;                   // scores: sigmoid or softmax of the logits; weights over their sum, or as they are
  float sum_eps;
};

// One warp per token; lane l holds experts l, l + 32, ...
__device__ __forceinline__ void route_select(const RouteArgs& a, const float* logits, int t) {
  const int lane = threadIdx.x & 31;
  float s[MOE_MAX_EXPERTS / 32], c[MOE_MAX_EXPERTS / 32], mx = -INFINITY, sum = 0.f;
#pragma unroll
  for (int j = 0; j < MOE_MAX_EXPERTS / 32; ++j) {
    const int e = lane + 32 * j;
    s[j] = e < a.E ? logits[e] : -INFINITY;
    mx = fmaxf(mx, s[j]);
  }
  if (a.sigmoid) {
    // without corrections the order of the logits is that of their scores, also where these have rounded to one
#pragma unroll
    for (int j = 0; j < MOE_MAX_EXPERTS / 32; ++j) {
      const int e = lane + 32 * j;
      const float z = s[j];
      s[j] = sigmoid_f(z);
      c[j] = e >= a.E ? -INFINITY : a.correction != nullptr ? s[j] + a.correction[e] : z;
    }
  } else {
    mx = warp_max(mx);
#pragma unroll
    for (int j = 0; j < MOE_MAX_EXPERTS / 32; ++j) {
      s[j] = expf(s[j] - mx);
      sum += s[j];
    }
    const float inv = 1.f / warp_sum(sum);
#pragma unroll
    for (int j = 0; j < MOE_MAX_EXPERTS / 32; ++j) {
      const int e = lane + 32 * j;
      s[j] *= inv;
      c[j] = e < a.E ? s[j] + (a.correction != nullptr ? a.correction[e] : 0.f) : -INFINITY;
    }
  }
  float total = 0.f, my_w = 0.f;
  int my_id = 0;
  for (int k = 0; k < a.topk; ++k) {
    float best = -INFINITY, score = 0.f;
    int id = MOE_MAX_EXPERTS;
#pragma unroll
    for (int j = 0; j < MOE_MAX_EXPERTS / 32; ++j)
      if (c[j] > best) { best = c[j]; id = lane + 32 * j; score = s[j]; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o), os = __shfl_xor_sync(0xffffffffu, score, o);
      const int oi = __shfl_xor_sync(0xffffffffu, id, o);
      if (ob > best || (ob == best && oi < id)) { best = ob; id = oi; score = os; }
    }
    if (id >= a.E) { id = 0; score = 0.f; }        // (scores that are not numbers: stay inside the experts)
#pragma unroll
    for (int j = 0; j < MOE_MAX_EXPERTS / 32; ++j)
      if (lane + 32 * j == id) c[j] = -INFINITY;
    total += score;
    if (lane == k) { my_w = score; my_id = id; }
  }
  if (lane < a.topk) {
    a.topk_w[static_cast<long long>(t) * a.topk + lane] = a.normalize ? my_w / (total + a.sum_eps) : my_w;
    a.topk_ids[static_cast<long long>(t) * a.topk + lane] = my_id;
  }
  if (lane < a.gates) a.gate[static_cast<long long>(t) * a.gates + lane] = sigmoid_f(logits[a.E + lane]);
}

// 16 MT tokens per CTA, the row dimension cut among the warps. A lane takes eight neighbouring elements of a token's row and
// the same eight of an expert's: the order of the row dimension inside a dot product is free, so two of its pairs are the low
// and high halves of one MMA's K and the other two of the next one's, and nothing passes through shared memory but the
// warps' partial sums.
template <int MT, int WARPS>
__global__ void __launch_bounds__(32 * WARPS)
moe_route_bf16_kernel(const RouteArgs a) {
  extern __shared__ float route_smem[];
  constexpr int ROWS = 16 * MT;
  float* part = route_smem;                        // [WARPS][ROWS][64]
  float* logits = route_smem + WARPS * ROWS * 64;  // [ROWS][n_out]
  const int n_out = a.E + a.gates;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gr = lane >> 2, gc = lane & 3;
  const int t0 = blockIdx.x * ROWS;
  const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(a.x);
  const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(a.w);
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  for (int n0 = 0; n0 < n_out; n0 += 64) {
    float acc[MT][8][4] = {};
    for (int k = warp * 32 + gc * 8; k - gc * 8 < a.H; k += WARPS * 32) {
      uint4 av[MT][2], bv[8];
      const bool kin = k < a.H;
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int t = t0 + m * 16 + h * 8 + gr;
          av[m][h] = kin && t < a.T ? *reinterpret_cast<const uint4*>(x + t * a.ldx + k) : zero;
        }
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int n = n0 + j * 8 + gr;
        bv[j] = kin && n < n_out ? *reinterpret_cast<const uint4*>(w + n * a.ldw + k) : zero;
      }
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const uint32_t lo[4] = {av[m][0].x, av[m][1].x, av[m][0].y, av[m][1].y};
        const uint32_t hi[4] = {av[m][0].z, av[m][1].z, av[m][0].w, av[m][1].w};
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          if (n0 + j * 8 >= n_out) continue;
          mma_bf16(acc[m][j], lo, bv[j].x, bv[j].y);
          mma_bf16(acc[m][j], hi, bv[j].z, bv[j].w);
        }
      }
    }
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int h = 0; h < 2; ++h)
          *reinterpret_cast<float2*>(part + (warp * ROWS + m * 16 + h * 8 + gr) * 64 + j * 8 + gc * 2) =
              make_float2(acc[m][j][2 * h], acc[m][j][2 * h + 1]);
    __syncthreads();
    for (int i = threadIdx.x; i < ROWS * 64; i += 32 * WARPS) {
      const int r = i >> 6, n = n0 + (i & 63);
      if (n >= n_out) continue;
      float v = 0.f;
#pragma unroll
      for (int p = 0; p < WARPS; ++p) v += part[p * ROWS * 64 + i];
      logits[r * n_out + n] = v;
    }
    __syncthreads();
  }
  for (int r = warp; r < ROWS && t0 + r < a.T; r += WARPS) route_select(a, logits + r * n_out, t0 + r);
}

__global__ void __launch_bounds__(256)
moe_route_f32_kernel(const RouteArgs a) {
  __shared__ float logits[MOE_MAX_EXPERTS + ROUTE_MAX_GATES];
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float* x = reinterpret_cast<const float*>(a.x) + t * a.ldx;
  for (int n = warp; n < a.E + a.gates; n += 8) {
    const float* w = reinterpret_cast<const float*>(a.w) + n * a.ldw;
    float v = 0.f;
    for (int k = lane; k < a.H; k += 32) v = fmaf(x[k], w[k], v);
    v = warp_sum(v);
    if (lane == 0) logits[n] = v;
  }
  __syncthreads();
  if (warp == 0) route_select(a, logits, t);
}

// Single CTA: histogram -> padded exclusive scan -> per-tile expert ids.
// meta[0] = number of 128-row tiles, meta[1] = padded row count.
__global__ void __launch_bounds__(1024)
moe_align_kernel(const int* __restrict__ topk_ids, int n_pairs, int E, int tile_rows,
                 int* __restrict__ expert_offsets, int* __restrict__ expert_cursor,
                 int* __restrict__ tile_expert, int max_tiles, int* __restrict__ meta) {
  __shared__ int counts[MOE_MAX_EXPERTS];
  __shared__ int offsets[MOE_MAX_EXPERTS + 1];
  for (int e = threadIdx.x; e < E; e += blockDim.x) counts[e] = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < n_pairs; i += blockDim.x) {
    const int e = topk_ids[i];
    if (e >= 0 && e < E) atomicAdd(&counts[e], 1);
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    int off = 0;
    for (int e = 0; e < E; ++e) {
      offsets[e] = off;
      off += (counts[e] + tile_rows - 1) / tile_rows * tile_rows;
    }
    offsets[E] = off;
    meta[0] = off / tile_rows;
    meta[1] = off;
  }
  __syncthreads();
  for (int e = threadIdx.x; e <= E; e += blockDim.x) {
    expert_offsets[e] = offsets[e];
    if (e < E) expert_cursor[e] = 0;
  }
  const int tiles = offsets[E] / tile_rows;
  for (int m = threadIdx.x; m < max_tiles; m += blockDim.x) {
    int ex = 0;
    if (m < tiles) {
      const int row = m * tile_rows;
      while (ex + 1 < E && offsets[ex + 1] <= row) ++ex;
    }
    tile_expert[m] = ex;
  }
}

// One CTA per (token, k) pair: claim a sorted row and copy the token's hidden row there.
__global__ void __launch_bounds__(256)
moe_scatter_kernel(const uint4* __restrict__ x, long long ldx, const int* __restrict__ topk_ids,
                   const float* __restrict__ topk_w, const int* __restrict__ expert_offsets,
                   int* __restrict__ expert_cursor, uint4* __restrict__ a_sorted,
                   float* __restrict__ row_scale, int* __restrict__ sorted_pos, int n_pairs, int topk,
                   int nvec, int E) {
  __shared__ int s_pos;
  for (int pair = blockIdx.x; pair < n_pairs; pair += gridDim.x) {
    if (threadIdx.x == 0) {
      const int e = topk_ids[pair];
      int pos = -1;
      if (e >= 0 && e < E) pos = expert_offsets[e] + atomicAdd(&expert_cursor[e], 1);
      s_pos = pos;
      sorted_pos[pair] = pos;
      if (pos >= 0) row_scale[pos] = topk_w[pair];
    }
    __syncthreads();
    const int pos = s_pos;
    if (pos >= 0) {
      const uint4* src = x + (pair / topk) * ldx;
      uint4* dst = a_sorted + static_cast<long long>(pos) * nvec;
      for (int v = threadIdx.x; v < nvec; v += blockDim.x) dst[v] = src[v];
    }
    __syncthreads();
  }
}

// out[t] = sum_k y[pos[t,k]] (+ gate[t] shared[t]; no gate: one) in fp32, rounded once.
template <typename T_>
__global__ void __launch_bounds__(256)
moe_combine_kernel(const T_* __restrict__ y, const int* __restrict__ sorted_pos, const T_* __restrict__ shared_y,
                   long long lds, const float* __restrict__ gate, T_* __restrict__ out, long long ldo, int T, int topk,
                   int H) {
  const int nvec = H >> 3;
  for (int t = blockIdx.x; t < T; t += gridDim.x) {
    for (int v = threadIdx.x; v < nvec; v += blockDim.x) {
      float acc[8], f[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[j] = 0.f;
      for (int k = 0; k < topk; ++k) {
        const int pos = sorted_pos[t * topk + k];
        if (pos < 0) continue;
        ld8(y + static_cast<long long>(pos) * H + v * 8, f);
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[j] += f[j];
      }
      if (shared_y != nullptr) {
        const float g = gate != nullptr ? gate[t] : 1.f;
        ld8(shared_y + t * lds + v * 8, f);
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[j] = fmaf(g, f[j], acc[j]);
      }
      st8(out + t * ldo + v * 8, acc);
    }
  }
}

static int moe_check(const char* what) {
  cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) {
    set_last_error("%s launch failed: %s", what, cudaGetErrorString(e));
    return 1;
  }
  return 0;
}

}  // namespace tw

using namespace tw;

extern "C" int tw_moe_router(const void* x, long long ldx, const void* wg, float* topk_w, int* topk_ids,
                             float* logits_out, int T, int H, int E, int topk, int renormalize,
                             cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H % 8 != 0 || ldx % 8 != 0 || topk < 1 || topk > MOE_MAX_TOPK || topk > E) {
    set_last_error("moe_router: unsupported shape (H=%d, E=%d, topk=%d)", H, E, topk);
    return 1;
  }
  const size_t smem = static_cast<size_t>(E) * H * 2;
  if (smem > 200 * 1024) {
    set_last_error("moe_router: gate weight (%zu bytes) does not fit in shared memory", smem);
    return 1;
  }
  const int cap = device_sm_count();
  auto xb = reinterpret_cast<const __nv_bfloat16*>(x);
  auto wb = reinterpret_cast<const __nv_bfloat16*>(wg);
  // tokens per warp: at most 64 accumulator registers per thread, room left for the prefetched row pieces
#define TW_ROUTER_CASE(NE, TPW)                                                                     \
  case NE: {                                                                                        \
    auto kern = moe_router_kernel<NE, TPW>;                                                         \
    int grid = (T + 16 * TPW - 1) / (16 * TPW);                                                     \
    if (grid > cap) grid = cap;                                                                     \
    cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)); \
    kern<<<grid, 512, smem, stream>>>(xb, ldx, wb, topk_w, topk_ids, logits_out, T, H, topk,         \
                                      renormalize);                                                 \
    break;                                                                                          \
  }
  switch (E) {
    TW_ROUTER_CASE(4, 4)
    TW_ROUTER_CASE(8, 2)
    TW_ROUTER_CASE(16, 1)
    TW_ROUTER_CASE(32, 1)
    default:
      set_last_error("moe_router: number of experts %d not in {4, 8, 16, 32}", E);
      return 1;
  }
#undef TW_ROUTER_CASE
  return moe_check("moe_router");
}

extern "C" int tw_moe_route(const void* x, long long ldx, const void* w, long long ldw, const float* correction,
                            float* topk_w, int* topk_ids, float* gate, int T, int H, int E, int gates, int topk,
                            int sigmoid, int normalize, float sum_eps, int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (E < 1 || E > MOE_MAX_EXPERTS || topk < 1 || topk > E || topk > ROUTE_MAX_TOPK || gates < 0 ||
      gates > ROUTE_MAX_GATES || (gates > 0 && gate == nullptr)) {
    set_last_error("moe_route: unsupported sizes (%d experts, top %d, %d gates)", E, topk, gates);
    return 1;
  }
  const RouteArgs a{x, ldx, w, ldw, correction, topk_w, topk_ids, gate, T, H, E, gates, topk, sigmoid, normalize, sum_eps};
  if (dtype != TW_BF16) {
    moe_route_f32_kernel<<<T, 256, 0, stream>>>(a);
    return moe_check("moe_route");
  }
  if (H % 8 != 0 || ldx % 8 != 0 || ldw % 8 != 0 || (reinterpret_cast<uintptr_t>(x) & 15) != 0 ||
      (reinterpret_cast<uintptr_t>(w) & 15) != 0) {
    set_last_error("moe_route: rows of %d elements on 16-byte boundaries are needed", H);
    return 1;
  }
#define TW_GO(MT, WARPS)                                                                                       \
  do {                                                                                                         \
    auto kern = moe_route_bf16_kernel<MT, WARPS>;                                                              \
    const int smem = (WARPS * 16 * MT * 64 + 16 * MT * (E + gates)) * 4;                                       \
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);       \
    if (e != cudaSuccess) {                                                                                    \
      set_last_error("moe_route: cudaFuncSetAttribute(smem=%d) failed: %s", smem, cudaGetErrorString(e));      \
      return 1;                                                                                                \
    }                                                                                                          \
    kern<<<(T + 16 * MT - 1) / (16 * MT), 32 * WARPS, smem, stream>>>(a);                                      \
  } while (0)
  if (T >= 32 * device_sm_count()) TW_GO(2, 8);
  else TW_GO(1, 16);
#undef TW_GO
  return moe_check("moe_route");
}

extern "C" int tw_moe_align(const int* topk_ids, int n_pairs, int E, int tile_rows, int* expert_offsets,
                            int* expert_cursor, int* tile_expert, int max_tiles, int* meta,
                            cudaStream_t stream) {
  if (E > MOE_MAX_EXPERTS) {
    set_last_error("moe_align: at most %d experts", MOE_MAX_EXPERTS);
    return 1;
  }
  moe_align_kernel<<<1, 1024, 0, stream>>>(topk_ids, n_pairs, E, tile_rows, expert_offsets, expert_cursor,
                                           tile_expert, max_tiles, meta);
  return moe_check("moe_align");
}

extern "C" int tw_moe_scatter(const void* x, long long ldx, const int* topk_ids, const float* topk_w,
                              const int* expert_offsets, int* expert_cursor, void* a_sorted,
                              float* row_scale, int* sorted_pos, int n_pairs, int topk, int H, int E, int dtype,
                              cudaStream_t stream) {
  if (n_pairs <= 0) return 0;
  const int per = dtype == TW_BF16 ? 8 : 4;          // elements in 16 bytes
  if (H % per != 0 || ldx % per != 0) {
    set_last_error("moe_scatter: rows of %d elements are not made of 16-byte pieces", H);
    return 1;
  }
  int grid = n_pairs;
  const int cap = device_sm_count() * 8;
  if (grid > cap) grid = cap;
  moe_scatter_kernel<<<grid, 256, 0, stream>>>(reinterpret_cast<const uint4*>(x), ldx / per, topk_ids, topk_w,
                                               expert_offsets, expert_cursor, reinterpret_cast<uint4*>(a_sorted),
                                               row_scale, sorted_pos, n_pairs, topk, H / per, E);
  return moe_check("moe_scatter");
}

// shared_y (or null): [T, H] with row stride lds, times gate [T] (or null: one).
extern "C" int tw_moe_combine(const void* y, const int* sorted_pos, const void* shared_y, long long lds, const float* gate,
                              void* out, long long ldo, int T, int topk, int H, int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H % 8 != 0 || ldo % 8 != 0 || lds % 8 != 0) {
    set_last_error("moe_combine: rows of %d elements (multiples of eight are needed)", H);
    return 1;
  }
  int grid = T;
  const int cap = device_sm_count() * 8;
  if (grid > cap) grid = cap;
#define TW_GO(TT)                                                                                                   \
  moe_combine_kernel<TT><<<grid, 256, 0, stream>>>(reinterpret_cast<const TT*>(y), sorted_pos,                      \
                                                   reinterpret_cast<const TT*>(shared_y), lds, gate,                \
                                                   reinterpret_cast<TT*>(out), ldo, T, topk, H)
  if (dtype == TW_BF16) TW_GO(__nv_bfloat16);
  else TW_GO(float);
#undef TW_GO
  return moe_check("moe_combine");
}
