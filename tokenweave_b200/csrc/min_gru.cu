// minGRU: a gated recurrence whose gates read the current token alone, channel by channel
//
//     z = sigmoid(pz + bz) ;  u = px + bx ;  S <- (1 - z) S + z (u >= 0 ? u + 1/2 : sigmoid(u)) ;  out = S silu(pg)
//
// on projected rows [pz | px | pg] of n channels each (a multiple of eight). The state is fp32 [slots, n], read for a
// sequence with tokens before the step's (zeros otherwise) and moved on; everything is computed in fp32.
//
//   scan   token by token, eight channels per thread: decoding and short runs
//   chunk  long runs, each row read once: a CTA owns CH channels of a sequence and walks over it in tiles of 256 tokens. A
//          thread takes two channels of eight consecutive tokens, whose steps compose to one, S -> A S + B; a warp
//          composes the 32 of a channel, in order, with the state before the tile, which gives every thread the state
//          its tokens start from. Tiles come through a ring of four in shared memory
#include "tw_common.cuh"
#include "tw_host.h"
#include "tw_kernels.h"
#include "tw_mma.cuh"
#include "tw_typed.cuh"

namespace tw {

struct GruArgs {
  const void* p; long long ldp;
  const float *bz, *bx;
  float* state;
  void* out; long long ldo;
  const int *seqs, *cu_q, *kv_lens, *slots;
  int n_seqs, n;
};

constexpr float NEG_LOG2E = -1.4426950408889634f;

// 1 / (1 + 2^x): the hardware's exponential and reciprocal, both good to 2^-22 (an infinite power gives zero)
__device__ __forceinline__ float2 gru_logistic(float2 x) {
  float2 e;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e.x) : "f"(x.x));
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e.y) : "f"(x.y));
  e = fma2(e, make_float2(1.f, 1.f), make_float2(1.f, 1.f));
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(e.x) : "f"(e.x));
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(e.y) : "f"(e.y));
  return e;
}

// Two channels: keep = 1 - z, add = z * candidate.
template <typename T>
__device__ __forceinline__ void gru_gates(float2 pz, float2 px, float2 bz, float2 bx, float2& keep, float2& add) {
  const float2 one = make_float2(1.f, 1.f), half = make_float2(0.5f, 0.5f), l = make_float2(NEG_LOG2E, NEG_LOG2E);
  const float2 u = fma2(px, one, bx);
  float2 z, c;
  if (sizeof(T) == 2) {
    z = gru_logistic(mul2(fma2(pz, one, bz), l));
    c = gru_logistic(mul2(u, l));
  } else {
    z = make_float2(sigmoid_f(pz.x + bz.x), sigmoid_f(pz.y + bz.y));
    c = make_float2(sigmoid_f(u.x), sigmoid_f(u.y));
  }
  const float2 lin = fma2(u, one, half);
  c.x = u.x >= 0.f ? lin.x : c.x;
  c.y = u.y >= 0.f ? lin.y : c.y;
  keep = fma2(z, make_float2(-1.f, -1.f), one);
  add = mul2(z, c);
}

template <typename T>
__device__ __forceinline__ float2 gru_output(float2 s, float2 g) {
  if (sizeof(T) == 2) return mul2(s, mul2(g, gru_logistic(mul2(g, make_float2(NEG_LOG2E, NEG_LOG2E)))));
  return make_float2(s.x * silu_f(g.x), s.y * silu_f(g.y));
}

__device__ __forceinline__ float2 ld2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 ld2(const __nv_bfloat16* p) { return unpack_bf16x2(*reinterpret_cast<const uint32_t*>(p)); }
__device__ __forceinline__ void st2(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
__device__ __forceinline__ void st2(__nv_bfloat16* p, float2 v) { *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(v.x, v.y); }

template <typename T>
__global__ void __launch_bounds__(256)
min_gru_scan_kernel(const GruArgs a) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (c >= a.n) return;
  const int b = a.seqs[blockIdx.y], t0 = a.cu_q[b], t1 = a.cu_q[b + 1];
  float* st = a.state + static_cast<long long>(a.slots[b]) * a.n + c;
  float s[8], bz[8], bx[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) s[j] = 0.f;
  if (a.kv_lens[b] > t1 - t0) ld8(st, s);
  ld8(a.bz + c, bz);
  ld8(a.bx + c, bx);
  for (int t = t0; t < t1; ++t) {
    const T* p = reinterpret_cast<const T*>(a.p) + t * a.ldp + c;
    float z[8], x[8], g[8];
    ld8(p, z);
    ld8(p + a.n, x);
    ld8(p + 2 * a.n, g);
#pragma unroll
    for (int j = 0; j < 8; j += 2) {
      float2 keep, add;
      gru_gates<T>(make_float2(z[j], z[j + 1]), make_float2(x[j], x[j + 1]), make_float2(bz[j], bz[j + 1]),
                   make_float2(bx[j], bx[j + 1]), keep, add);
      const float2 v = fma2(keep, make_float2(s[j], s[j + 1]), add);
      const float2 o = gru_output<T>(v, make_float2(g[j], g[j + 1]));
      s[j] = v.x;
      s[j + 1] = v.y;
      g[j] = o.x;
      g[j + 1] = o.y;
    }
    st8(reinterpret_cast<T*>(a.out) + t * a.ldo + c, g);
  }
  st8(st, s);
}

constexpr int GRU_SEG = 8, GRU_SEGS = 32, GRU_TILE = GRU_SEG * GRU_SEGS, GRU_STAGES = 4;

// The rows of a tile in shared memory, one part of the projection behind the other. Threads of a warp that read the same
// channels stand eight rows apart: rows that share 128 bytes change places from eight to eight, so that these threads meet
// different banks.
template <typename T, int CH>
struct GruSmem {
  static constexpr int ROW = CH * sizeof(T), PART = GRU_TILE * ROW, STAGE = 3 * PART;
  static constexpr int SUMS = GRU_SEGS * (CH + 1) * 4;
  static constexpr int TOTAL = GRU_STAGES * STAGE + 2 * SUMS;
  static __device__ __forceinline__ int row(int r) { return (r ^ ((r >> 3) & (128 / ROW - 1))) * ROW; }
};

template <typename T, int CH>
__global__ void __launch_bounds__(CH * 16)
min_gru_chunk_kernel(const GruArgs a) {
  using S = GruSmem<T, CH>;
  constexpr int LANES = CH / 2, THREADS = CH * 16;           // threads that share a segment; of the CTA
  constexpr int PIECES = S::ROW / 16, PER = 16 / sizeof(T);  // 16-byte pieces of a row, channels of a piece
  extern __shared__ __align__(16) uint8_t gru_smem[];
  float* a_s = reinterpret_cast<float*>(gru_smem + GRU_STAGES * S::STAGE);       // [GRU_SEGS][CH + 1]
  float* b_s = a_s + GRU_SEGS * (CH + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seg = threadIdx.x / LANES, cc = (threadIdx.x % LANES) * 2;
  const int c0 = blockIdx.x * CH, c = c0 + cc;
  const bool mine = c < a.n;                                 // (n is even)
  const int b = a.seqs[blockIdx.y], t0 = a.cu_q[b], len = a.cu_q[b + 1] - t0;
  const bool past = a.kv_lens[b] > len;
  float* state = a.state + static_cast<long long>(a.slots[b]) * a.n + c0;
  const T* p = reinterpret_cast<const T*>(a.p) + t0 * a.ldp + c0;
  T* out = reinterpret_cast<T*>(a.out) + t0 * a.ldo + c;
  const float2 bz = mine ? ld2(a.bz + c) : make_float2(0.f, 0.f), bx = mine ? ld2(a.bx + c) : make_float2(0.f, 0.f);
  // the state before the tile, of the two channels that this warp composes (the same in every lane)
  float carry[2];
#pragma unroll
  for (int k = 0; k < 2; ++k) carry[k] = past && c0 + 2 * warp + k < a.n ? state[2 * warp + k] : 0.f;

  const int tiles = (len + GRU_TILE - 1) / GRU_TILE;
  auto request = [&](int tile) {                             // (what lies outside comes as zeros)
    uint8_t* dst = gru_smem + (tile % GRU_STAGES) * S::STAGE;
    for (int i = threadIdx.x; i < GRU_TILE * PIECES; i += THREADS) {
      const int r = i / PIECES, piece = i % PIECES, t = tile * GRU_TILE + r;
      const bool there = t < len && c0 + piece * PER < a.n;
      const T* src = there ? p + t * a.ldp + piece * PER : reinterpret_cast<const T*>(a.p);
      uint8_t* to = dst + S::row(r) + piece * 16;
#pragma unroll
      for (int part = 0; part < 3; ++part)
        cp_async16(to + part * S::PART, there ? src + part * static_cast<long long>(a.n) : src, there ? 16 : 0);
    }
  };
  for (int tile = 0; tile < GRU_STAGES - 1; ++tile) {
    if (tile < tiles) request(tile);
    cp_async_commit();
  }
  for (int tile = 0; tile < tiles; ++tile) {
    cp_async_wait<GRU_STAGES - 2>();
    __syncthreads();                                         // the tile is there, and everyone is done with the last one
    if (tile + GRU_STAGES - 1 < tiles) request(tile + GRU_STAGES - 1);
    cp_async_commit();
    const uint8_t* rows = gru_smem + (tile % GRU_STAGES) * S::STAGE + cc * sizeof(T);
    const int first = tile * GRU_TILE + seg * GRU_SEG;
    float2 keep[GRU_SEG], add[GRU_SEG];
    float2 A = make_float2(1.f, 1.f), B = make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < GRU_SEG; ++i) {
      const uint8_t* at = rows + S::row(seg * GRU_SEG + i);
      gru_gates<T>(ld2(reinterpret_cast<const T*>(at)), ld2(reinterpret_cast<const T*>(at + S::PART)), bz, bx, keep[i], add[i]);
      if (first + i >= len) {                                // behind the last token: nothing changes
        keep[i] = make_float2(1.f, 1.f);
        add[i] = make_float2(0.f, 0.f);
      }
      A = mul2(A, keep[i]);
      B = fma2(keep[i], B, add[i]);
    }
    float* sa = a_s + seg * (CH + 1) + cc;
    float* sb = b_s + seg * (CH + 1) + cc;
    sa[0] = A.x;
    sa[1] = A.y;
    sb[0] = B.x;
    sb[1] = B.y;
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      // lane: segment. Composition of the segments up to this one
      const int at = lane * (CH + 1) + 2 * warp + k;
      float ca = a_s[at], cb = b_s[at];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float pa = __shfl_up_sync(0xffffffffu, ca, o), pb = __shfl_up_sync(0xffffffffu, cb, o);
        if (lane >= o) {
          cb = fmaf(ca, pb, cb);
          ca *= pa;
        }
      }
      const float behind = fmaf(ca, carry[k], cb);           // the state behind this segment
      const float before = __shfl_up_sync(0xffffffffu, behind, 1);
      b_s[at] = lane == 0 ? carry[k] : before;
      carry[k] = __shfl_sync(0xffffffffu, behind, 31);
    }
    __syncthreads();
    float2 s = make_float2(sb[0], sb[1]);
#pragma unroll
    for (int i = 0; i < GRU_SEG; ++i) {
      s = fma2(keep[i], s, add[i]);
      const float2 g = ld2(reinterpret_cast<const T*>(rows + 2 * S::PART + S::row(seg * GRU_SEG + i)));
      if (mine && first + i < len) st2(out + (first + i) * a.ldo, gru_output<T>(s, g));
    }
  }
  if (lane == 0) {
#pragma unroll
    for (int k = 0; k < 2; ++k)
      if (c0 + 2 * warp + k < a.n) state[2 * warp + k] = carry[k];
  }
}

template <typename T, int CH>
static int launch_gru_chunk(const GruArgs& a, cudaStream_t stream) {
  auto kern = min_gru_chunk_kernel<T, CH>;
  constexpr int smem = GruSmem<T, CH>::TOTAL;
  const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) {
    set_last_error("min_gru: cudaFuncSetAttribute(smem=%d) failed: %s", smem, cudaGetErrorString(e));
    return 1;
  }
  kern<<<dim3((a.n + CH - 1) / CH, a.n_seqs), CH * 16, smem, stream>>>(a);
  return 0;
}

static bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace tw

using namespace tw;

// chunked: 0 token by token, 1 tiles
extern "C" int tw_min_gru(const void* p, long long ldp, const float* bz, const float* bx, float* state, void* out,
                          long long ldo, const int* seqs, int n_seqs, const int* cu_q, const int* kv_lens, const int* slots,
                          int n, int chunked, int dtype, cudaStream_t stream) {
  if (n_seqs <= 0 || n <= 0) return 0;
  if (n % 8 != 0 || ldp % 8 != 0 || ldo % 8 != 0 || ldp < 3LL * n || ldo < n || n_seqs > 65535 || !aligned16(p) ||
      !aligned16(bz) || !aligned16(bx) || !aligned16(state) || !aligned16(out)) {
    set_last_error("min_gru: %d channels of %d sequences: multiples of eight on 16-byte boundaries are needed", n, n_seqs);
    return 1;
  }
  const GruArgs a{p, ldp, bz, bx, state, out, ldo, seqs, cu_q, kv_lens, slots, n_seqs, n};
  if (chunked) {
    // channels per CTA: enough CTAs for the machine
    const bool narrow = static_cast<long long>((n + 31) / 32) * n_seqs < device_sm_count() * 3 / 4;
    if (dtype != TW_BF16 ? launch_gru_chunk<float, 16>(a, stream)
        : narrow         ? launch_gru_chunk<__nv_bfloat16, 16>(a, stream)
                         : launch_gru_chunk<__nv_bfloat16, 32>(a, stream))
      return 1;
  } else {
    int threads = (n / 8 + 31) / 32 * 32;
    if (threads > 128) threads = 128;
    const dim3 grid((n / 8 + threads - 1) / threads, n_seqs);
    if (dtype == TW_BF16) min_gru_scan_kernel<__nv_bfloat16><<<grid, threads, 0, stream>>>(a);
    else min_gru_scan_kernel<float><<<grid, threads, 0, stream>>>(a);
  }
  const cudaError_t e = cudaGetLastError();
  if (e == cudaSuccess) return 0;
  set_last_error("min_gru launch failed: %s", cudaGetErrorString(e));
  return 1;
}
