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
//          its tokens start from. The next tile's rows are requested before this one's are worked on
#include "tw_host.h"
#include "tw_kernels.h"
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

// keep = 1 - z, add = z * candidate
template <typename T>
__device__ __forceinline__ void gru_gates(float pz, float px, float& keep, float& add) {
  const float z = sigmoid_t<T>(pz);
  keep = 1.f - z;
  add = z * (px >= 0.f ? px + 0.5f : sigmoid_t<T>(px));
}

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
    for (int j = 0; j < 8; ++j) {
      float keep, add;
      gru_gates<T>(z[j] + bz[j], x[j] + bx[j], keep, add);
      s[j] = fmaf(keep, s[j], add);
      g[j] = s[j] * silu_t<T>(g[j]);
    }
    st8(reinterpret_cast<T*>(a.out) + t * a.ldo + c, g);
  }
  st8(st, s);
}

template <typename T>
struct __align__(2 * sizeof(T)) Pair {
  T x, y;
};

constexpr int GRU_SEG = 8, GRU_SEGS = 32, GRU_TILE = GRU_SEG * GRU_SEGS;

template <typename T, int CH>
__global__ void __launch_bounds__(CH * 16, 32 / CH)
min_gru_chunk_kernel(const GruArgs a) {
  constexpr int LANES = CH / 2;                              // threads that share a segment
  __shared__ float a_s[2][GRU_SEGS][CH + 1], b_s[2][GRU_SEGS][CH + 1];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seg = threadIdx.x / LANES, cc = (threadIdx.x % LANES) * 2;
  const int c0 = blockIdx.x * CH, c = c0 + cc;
  const bool mine = c < a.n;                                 // (n is even)
  const int b = a.seqs[blockIdx.y], t0 = a.cu_q[b], len = a.cu_q[b + 1] - t0;
  const bool past = a.kv_lens[b] > len;
  float* state = a.state + static_cast<long long>(a.slots[b]) * a.n + c0;
  const T* p = reinterpret_cast<const T*>(a.p) + t0 * a.ldp + c;
  T* out = reinterpret_cast<T*>(a.out) + t0 * a.ldo + c;
  const float2 bz = mine ? make_float2(a.bz[c], a.bz[c + 1]) : make_float2(0.f, 0.f);
  const float2 bx = mine ? make_float2(a.bx[c], a.bx[c + 1]) : make_float2(0.f, 0.f);
  // the state before the tile, of the two channels that this warp composes (the same in every lane)
  float carry[2];
#pragma unroll
  for (int k = 0; k < 2; ++k) carry[k] = past && c0 + 2 * warp + k < a.n ? state[2 * warp + k] : 0.f;

  Pair<T> z[GRU_SEG], x[GRU_SEG], g[GRU_SEG];
  auto request = [&](int first) {
#pragma unroll
    for (int i = 0; i < GRU_SEG; ++i) {
      const int t = first + seg * GRU_SEG + i;
      if (!mine || t >= len) continue;
      const T* row = p + t * a.ldp;
      z[i] = *reinterpret_cast<const Pair<T>*>(row);
      x[i] = *reinterpret_cast<const Pair<T>*>(row + a.n);
      g[i] = *reinterpret_cast<const Pair<T>*>(row + 2 * a.n);
    }
  };
  request(0);
  for (int first = 0, buf = 0; first < len; first += GRU_TILE, buf ^= 1) {
    float2 keep[GRU_SEG], add[GRU_SEG];
    Pair<T> gate[GRU_SEG];
    float2 A = make_float2(1.f, 1.f), B = make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < GRU_SEG; ++i) {
      const int t = first + seg * GRU_SEG + i;
      if (!mine || t >= len) {                               // behind the last token: nothing changes
        keep[i] = make_float2(1.f, 1.f);
        add[i] = make_float2(0.f, 0.f);
        continue;
      }
      gru_gates<T>(ld1(&z[i].x) + bz.x, ld1(&x[i].x) + bx.x, keep[i].x, add[i].x);
      gru_gates<T>(ld1(&z[i].y) + bz.y, ld1(&x[i].y) + bx.y, keep[i].y, add[i].y);
      gate[i] = g[i];
      A = make_float2(A.x * keep[i].x, A.y * keep[i].y);
      B = make_float2(fmaf(keep[i].x, B.x, add[i].x), fmaf(keep[i].y, B.y, add[i].y));
    }
    if (first + GRU_TILE < len) request(first + GRU_TILE);
    a_s[buf][seg][cc] = A.x;
    a_s[buf][seg][cc + 1] = A.y;
    b_s[buf][seg][cc] = B.x;
    b_s[buf][seg][cc + 1] = B.y;
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      // lane: segment. Composition of the segments up to this one
      float ca = a_s[buf][lane][2 * warp + k], cb = b_s[buf][lane][2 * warp + k];
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
      b_s[buf][lane][2 * warp + k] = lane == 0 ? carry[k] : before;
      carry[k] = __shfl_sync(0xffffffffu, behind, 31);
    }
    __syncthreads();
    float2 s = make_float2(b_s[buf][seg][cc], b_s[buf][seg][cc + 1]);
#pragma unroll
    for (int i = 0; i < GRU_SEG; ++i) {
      const int t = first + seg * GRU_SEG + i;
      if (!mine || t >= len) continue;
      s = make_float2(fmaf(keep[i].x, s.x, add[i].x), fmaf(keep[i].y, s.y, add[i].y));
      Pair<T> o;
      st1(&o.x, s.x * silu_t<T>(ld1(&gate[i].x)));
      st1(&o.y, s.y * silu_t<T>(ld1(&gate[i].y)));
      *reinterpret_cast<Pair<T>*>(out + t * a.ldo) = o;
    }
  }
  if (lane == 0) {
#pragma unroll
    for (int k = 0; k < 2; ++k)
      if (c0 + 2 * warp + k < a.n) state[2 * warp + k] = carry[k];
  }
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
#define TW_GO(T, CH) min_gru_chunk_kernel<T, CH><<<dim3((n + CH - 1) / CH, n_seqs), CH * 16, 0, stream>>>(a)
    if (dtype == TW_BF16) {
      if (narrow) TW_GO(__nv_bfloat16, 16); else TW_GO(__nv_bfloat16, 32);
    } else {
      if (narrow) TW_GO(float, 16); else TW_GO(float, 32);
    }
#undef TW_GO
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
