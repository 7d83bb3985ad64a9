// Residual blocks with a norm in front of a sublayer and one behind it, and averages over the depth of the network:
//
//     x <- x + N_post(sublayer(N_pre(x)))                       after every sublayer
//     X_n = x ;  x <- sum_{j <= n} coef[j] X_j                  after every layer (X_0: the embedding output)
//
//   tw_embed_sandwich  x = X_0 = scale * table[id] ; xa = N(x) (the first sublayer's input)
//   tw_sandwich_step   what lies between two sublayers, in one pass: norm of the sublayer's output, sum, (the layer's result
//                      kept, the average over all results so far,) and the next sublayer's norm (or the final one)
//
// N is a layer norm (mean taken off, weight and bias) or an RMS norm (weight alone). The stream and the kept results are
// fp32, y, xa and the norms' weights bf16 or fp32, all arithmetic is fp32; deviations are summed from the mean, not as a
// difference of squares. One CTA per row; the row stays in registers between the passes.
#include "tw_host.h"
#include "tw_kernels.h"
#include "tw_typed.cuh"

namespace tw {

struct SandwichArgs {
  const void* y; long long ldy;                  // [rows, H] sublayer output
  float* x; long long ldx;                       // [rows, H] stream
  int store;                                     // the new stream is written back
  const void *w_post, *b_post;                   // norm of the output
  const float* past; long long ldp, lds;         // X_j of row t: past + j * lds + t * ldp
  int n_past;
  const float* coef;                             // [n_past + 1]; null: no average
  float* result;                                 // X_n (row stride ldp); null: not kept
  const void *w_next, *b_next;                   // the next norm
  void* xa; long long lda;
  int rows, H, center;
  float eps;
  const int* ids; const void* table; long long ldt; int vocab; float scale;        // embedding
};

// Eight elements of a row from i on of which n are inside it. FULL: every thread's groups are (the row is as long as the CTA).
template <bool FULL, typename T>
__device__ __forceinline__ void ldg8(const T* p, int n, float (&v)[8]) {
  if (FULL) ld8(p, v);
  else ld8n<true>(p, n, v);
}
template <bool FULL, typename T>
__device__ __forceinline__ void stg8(T* p, int n, const float (&v)[8]) {
  if (FULL) st8(p, v);
  else st8n<true>(p, n, v);
}

// Block-wide mean and sum of squared deviations of a row in one exchange: every warp takes the deviations from its own mean, and
// the warps' results are put together with the distances between their means. Without `center` the mean is zero.
template <int VPT, bool FULL>
__device__ __forceinline__ void row_moments(const SandwichArgs& a, const float (&v)[VPT][8], float* scratch, float& mean,
                                            float& dev) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  // elements of the row that a warp holds
  auto held = [&](int w) {
    if (FULL) return 256.f * VPT;
    int n = 0;
#pragma unroll
    for (int k = 0; k < VPT; ++k) n += max(0, min(256, a.H - (w * 32 + k * static_cast<int>(blockDim.x)) * 8));
    return static_cast<float>(n);
  };
  float s = 0.f, m = 0.f;
  if (a.center) {
#pragma unroll
    for (int k = 0; k < VPT; ++k)
#pragma unroll
      for (int j = 0; j < 8; ++j) s += v[k][j];
    s = warp_sum(s);
    const float n = held(warp);
    m = n > 0.f ? s / n : 0.f;
  }
  float d = 0.f;
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int n = a.H - (threadIdx.x + k * blockDim.x) * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const float e = FULL || j < n ? v[k][j] - m : 0.f;
      d = fmaf(e, e, d);
    }
  }
  d = warp_sum(d);
  if (lane == 0) {
    scratch[warp] = s;
    scratch[32 + warp] = d;
  }
  __syncthreads();
  s = lane < warps ? scratch[lane] : 0.f;
  d = lane < warps ? scratch[32 + lane] : 0.f;
  mean = 0.f;
  if (a.center) {
    const float n = lane < warps ? held(lane) : 0.f;
    mean = warp_sum(s) / static_cast<float>(a.H);
    const float e = n > 0.f ? s / n - mean : 0.f;
    d = fmaf(n * e, e, d);
  }
  dev = warp_sum(d);
}

// Replaces a row by its norm. Elements outside the row are zeros. (Consecutive calls take different scratch.)
template <typename T, int VPT, bool FULL>
__device__ __forceinline__ void norm_row(const SandwichArgs& a, float (&v)[VPT][8], const void* w, const void* b,
                                         float* scratch) {
  float mean, dev;
  row_moments<VPT, FULL>(a, v, scratch, mean, dev);
  const float r = 1.f / sqrtf(dev / static_cast<float>(a.H) + a.eps);
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = (threadIdx.x + k * blockDim.x) * 8, n = a.H - i;
    if (!FULL && n <= 0) continue;
    float g[8], c[8];
    ldg8<FULL>(reinterpret_cast<const T*>(w) + i, n, g);
    if (b != nullptr) {
      ldg8<FULL>(reinterpret_cast<const T*>(b) + i, n, c);
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) c[j] = 0.f;
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) v[k][j] = fmaf((v[k][j] - mean) * r, g[j], c[j]);
  }
}

template <typename T, int VPT, bool FULL>
__device__ __forceinline__ void next_input(const SandwichArgs& a, int t, float (&v)[VPT][8], float* scratch) {
  norm_row<T, VPT, FULL>(a, v, a.w_next, a.b_next, scratch);
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = (threadIdx.x + k * blockDim.x) * 8, n = a.H - i;
    if (FULL || n > 0) stg8<FULL>(reinterpret_cast<T*>(a.xa) + t * a.lda + i, n, v[k]);
  }
}

template <typename T, int VPT, bool FULL, bool AVERAGE>
__global__ void __launch_bounds__(512)
sandwich_step_kernel(const SandwichArgs a) {
  __shared__ float scratch[2][64];
  const float own = AVERAGE ? a.coef[a.n_past] : 1.f;
  Raw8<T> y[VPT];
  float x[VPT][8];
  auto request = [&](int t) {
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (threadIdx.x + k * blockDim.x) * 8, n = a.H - i;
      y[k] = ld8raw<true>(reinterpret_cast<const T*>(a.y) + t * a.ldy + (FULL || n > 0 ? i : 0), FULL ? 8 : n);
      if (FULL || n > 0) ldg8<FULL>(a.x + t * a.ldx + i, n, x[k]);
    }
  };
  if (static_cast<int>(blockIdx.x) < a.rows) request(blockIdx.x);
  for (int t = blockIdx.x; t < a.rows; t += gridDim.x) {
    float v[VPT][8], sum[VPT][8];
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        v[k][j] = ld1(&y[k].v[j]);
        sum[k][j] = 0.f;
      }
      if (!AVERAGE) continue;
      const int i = (threadIdx.x + k * blockDim.x) * 8, n = a.H - i;
      if (!FULL && n <= 0) continue;
      const float* p = a.past + t * a.ldp + i;
#pragma unroll 4
      for (int q = 0; q < a.n_past; ++q) {
        const float c = a.coef[q];
        float u[8];
        ldg8<FULL>(p + q * a.lds, n, u);
#pragma unroll
        for (int j = 0; j < 8; ++j) sum[k][j] = fmaf(c, u[j], sum[k][j]);
      }
    }
    norm_row<T, VPT, FULL>(a, v, a.w_post, a.b_post, scratch[0]);
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (threadIdx.x + k * blockDim.x) * 8, n = a.H - i;
      if (!FULL && n <= 0) {
#pragma unroll
        for (int j = 0; j < 8; ++j) v[k][j] = 0.f;
        continue;
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) v[k][j] += x[k][j];
      if (AVERAGE) {
        if (a.result != nullptr) stg8<FULL>(a.result + t * a.ldp + i, n, v[k]);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[k][j] = fmaf(own, v[k][j], sum[k][j]);
      }
      if (a.store) stg8<FULL>(a.x + t * a.ldx + i, n, v[k]);
    }
    // the next row is on its way while this one's second norm is formed
    if (t + static_cast<int>(gridDim.x) < a.rows) request(t + gridDim.x);
    next_input<T, VPT, FULL>(a, t, v, scratch[1]);
  }
}

template <typename T, int VPT, bool FULL>
__global__ void __launch_bounds__(512)
embed_sandwich_kernel(const SandwichArgs a) {
  __shared__ float scratch[2][64];
  for (int t = blockIdx.x, turn = 0; t < a.rows; t += gridDim.x, turn ^= 1) {
    const int id = a.ids[t];
    const bool ok = id >= 0 && id < a.vocab;
    const T* src = reinterpret_cast<const T*>(a.table) + (ok ? id : 0) * a.ldt;
    float v[VPT][8];
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (threadIdx.x + k * blockDim.x) * 8, n = a.H - i;
#pragma unroll
      for (int j = 0; j < 8; ++j) v[k][j] = 0.f;
      if (!FULL && n <= 0) continue;
      if (ok) ldg8<FULL>(src + i, n, v[k]);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[k][j] *= a.scale;
      stg8<FULL>(a.x + t * a.ldx + i, n, v[k]);
      if (a.result != nullptr) stg8<FULL>(a.result + t * a.ldp + i, n, v[k]);
    }
    next_input<T, VPT, FULL>(a, t, v, scratch[turn]);
  }
}

static bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename T, int VPT, bool FULL>
static void launch_sandwich(const SandwichArgs& a, int threads, cudaStream_t stream) {
  // as many CTAs as fit at a time, so that each one's next row is on its way
  const int cap = device_sm_count() * (a.ids != nullptr ? 3 : 2) * (threads <= 128 ? 4 : threads <= 256 ? 2 : 1);
  const int grid = a.rows < cap ? a.rows : cap;
  if (a.ids != nullptr) embed_sandwich_kernel<T, VPT, FULL><<<grid, threads, 0, stream>>>(a);
  else if (a.coef != nullptr) sandwich_step_kernel<T, VPT, FULL, true><<<grid, threads, 0, stream>>>(a);
  else sandwich_step_kernel<T, VPT, FULL, false><<<grid, threads, 0, stream>>>(a);
}

static int run_sandwich(const SandwichArgs& a, int dtype, const char* what, cudaStream_t stream) {
  const int nvec = (a.H + 7) / 8, vpt = nvec <= 512 ? 1 : nvec <= 1024 ? 2 : 4;
  const int threads = ((nvec + vpt - 1) / vpt + 31) / 32 * 32;
  if (a.H <= 0 || threads > 512) {
    set_last_error("%s: rows of %d elements (up to 16384)", what, a.H);
    return 1;
  }
  if (a.ldy % 8 != 0 || a.ldx % 8 != 0 || a.lda % 8 != 0 || a.ldt % 8 != 0 || a.ldp % 8 != 0 || a.lds % 8 != 0 ||
      !aligned16(a.y) || !aligned16(a.x) || !aligned16(a.xa) || !aligned16(a.table) || !aligned16(a.past) ||
      !aligned16(a.result) || !aligned16(a.w_post) || !aligned16(a.b_post) || !aligned16(a.w_next) || !aligned16(a.b_next)) {
    set_last_error("%s: rows on 16-byte boundaries are needed", what);
    return 1;
  }
  const bool full = a.H == threads * vpt * 8;
#define TW_GO(TT)                                                                              \
  do {                                                                                         \
    if (vpt == 1 && full) launch_sandwich<TT, 1, true>(a, threads, stream);              \
    else if (vpt == 1) launch_sandwich<TT, 1, false>(a, threads, stream);                \
    else if (vpt == 2 && full) launch_sandwich<TT, 2, true>(a, threads, stream);         \
    else if (vpt == 2) launch_sandwich<TT, 2, false>(a, threads, stream);                \
    else launch_sandwich<TT, 4, false>(a, threads, stream);                              \
  } while (0)
  if (dtype == TW_BF16) TW_GO(__nv_bfloat16);
  else TW_GO(float);
#undef TW_GO
  const cudaError_t e = cudaGetLastError();
  if (e == cudaSuccess) return 0;
  set_last_error("%s launch failed: %s", what, cudaGetErrorString(e));
  return 1;
}

}  // namespace tw

using namespace tw;

extern "C" int tw_embed_sandwich(const int* ids, const void* table, long long ldt, int vocab, float scale, float* x,
                                 long long ldx, float* first, long long ldp, const void* w, const void* b, int center,
                                 void* xa, long long lda, int T, int H, float eps, int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  SandwichArgs a{};
  a.ids = ids; a.table = table; a.ldt = ldt; a.vocab = vocab; a.scale = scale;
  a.x = x; a.ldx = ldx; a.result = first; a.ldp = ldp; a.w_next = w; a.b_next = b; a.center = center;
  a.xa = xa; a.lda = lda; a.rows = T; a.H = H; a.eps = eps;
  return run_sandwich(a, dtype, "embed_sandwich", stream);
}

extern "C" int tw_sandwich_step(const void* y, long long ldy, float* x, long long ldx, int store, const void* w_post,
                                const void* b_post, const float* past, long long ldp, long long lds, int n_past,
                                const float* coef, float* result, const void* w_next, const void* b_next, int center,
                                void* xa, long long lda, int T, int H, float eps, int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (n_past < 0 || (coef != nullptr && n_past > 0 && past == nullptr)) {
    set_last_error("sandwich_step: an average over %d earlier results that are not there", n_past);
    return 1;
  }
  SandwichArgs a{};
  a.y = y; a.ldy = ldy; a.x = x; a.ldx = ldx; a.store = store; a.w_post = w_post; a.b_post = b_post;
  a.past = past; a.ldp = ldp; a.lds = lds; a.n_past = n_past; a.coef = coef; a.result = result;
  a.w_next = w_next; a.b_next = b_next; a.center = center;
  a.xa = xa; a.lda = lda; a.rows = T; a.H = H; a.eps = eps;
  return run_sandwich(a, dtype, "sandwich_step", stream);
}
