// Hyper-connections: the residual stream is S parallel fp32 rows per token. A sublayer reads one weighted sum of them and
// every stream is then rebuilt from all old ones and the sublayer's output:
//
//     u = sum_s in[s] x_s ;   y = sublayer(rmsnorm(u)) ;   x_t <- sum_s mix[s, t] x_s + mult out[t] y
//
//   tw_embed_streams   x_0 = table[id] (every stream begins as that row, it is stored once) ; xa = rmsnorm(sum_s in[s] x_0)
//                      (offset + w)
//   tw_streams_step    what lies between two sublayers, in one pass: the streams behind a sublayer's output and the next
//                      sublayer's normed input (behind the last one: the norm of the plain sum, the streams are not stored;
//                      behind the first one all old streams are read from the first)
//
// One CTA per row; the weighted sum stays in registers between the two passes (in shared memory beyond four streams). All
// arithmetic is fp32; y, w and xa are bf16 or fp32. S = 1 with coefficients of one is a pre-norm residual stream.
#include "tw_host.h"
#include "tw_kernels.h"
#include "tw_typed.cuh"

namespace tw {

constexpr int STREAMS_MAX = 16;

struct StreamsArgs {
  const void* y; long long ldy;                 // [rows, H] sublayer output
  float* x; long long ldx, lds;                 // stream s of row t: x + t * ldx + s * lds
  const float *mix, *out, *in;                  // [S, S] (from, to), [S], [S]; in null: all ones
  float mult;
  const void* w; float offset;                  // norm weight: offset + w
  void* xa; long long lda;
  int rows, H, S, store;
  long long ldr;                                // between old streams: lds, or 0 where all are the first
  float eps;
  // embedding
  const int* ids; const void* table; long long ldt; int vocab;
};

template <typename T, int VPT>
__device__ __forceinline__ void streams_norm(const StreamsArgs& a, int t, float (&u)[VPT][8], float ss, float* scratch) {
  float s[1] = {ss};
  block_sum<1>(s, scratch);
  const float r = 1.f / sqrtf(s[0] / static_cast<float>(a.H) + a.eps);
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = (threadIdx.x + k * blockDim.x) * 8;
    if (i >= a.H) continue;
    float g[8];
    ld8n<true>(reinterpret_cast<const T*>(a.w) + i, a.H - i, g);
#pragma unroll
    for (int j = 0; j < 8; ++j) g[j] = u[k][j] * r * (a.offset + g[j]);
    st8n<true>(reinterpret_cast<T*>(a.xa) + t * a.lda + i, a.H - i, g);
  }
}

template <typename T, int VPT, int SMAX>
__global__ void __launch_bounds__(512)
streams_step_kernel(const StreamsArgs a) {
  __shared__ float scratch[32];
  __shared__ float mix_s[SMAX * SMAX], out_s[SMAX], in_s[SMAX];      // mix_s[to][from]
  for (int i = threadIdx.x; i < a.S * a.S; i += blockDim.x) mix_s[(i % a.S) * SMAX + i / a.S] = a.mix[i];
  if (threadIdx.x < a.S) {
    out_s[threadIdx.x] = a.mult * a.out[threadIdx.x];
    in_s[threadIdx.x] = a.in != nullptr ? a.in[threadIdx.x] : 1.f;
  }
  __syncthreads();
  for (int t = blockIdx.x; t < a.rows; t += gridDim.x) {
    float u[VPT][8], ss = 0.f;
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (threadIdx.x + k * blockDim.x) * 8, n = a.H - i;
#pragma unroll
      for (int j = 0; j < 8; ++j) u[k][j] = 0.f;
      if (n <= 0) continue;
      float* x = a.x + t * a.ldx + i;
      float old[SMAX][8], y[8];
#pragma unroll
      for (int s = 0; s < SMAX; ++s)
        if (s < a.S) ld8n<true>(x + s * a.ldr, n, old[s]);
      ld8n<true>(reinterpret_cast<const T*>(a.y) + t * a.ldy + i, n, y);
#pragma unroll
      for (int to = 0; to < SMAX; ++to) {
        if (to >= a.S) continue;
        float v[8];
        const float o = out_s[to], in = in_s[to];
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = o * y[j];
#pragma unroll
        for (int s = 0; s < SMAX; ++s) {
          if (s >= a.S) continue;
          const float m = mix_s[to * SMAX + s];
#pragma unroll
          for (int j = 0; j < 8; ++j) v[j] = fmaf(m, old[s][j], v[j]);
        }
        if (a.store) st8n<true>(x + to * a.lds, n, v);
#pragma unroll
        for (int j = 0; j < 8; ++j) u[k][j] = fmaf(in, v[j], u[k][j]);
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += u[k][j] * u[k][j];
    }
    streams_norm<T, VPT>(a, t, u, ss, scratch);
  }
}

// More streams than a thread can hold eight elements of: four elements at a time.
template <typename T>
__global__ void __launch_bounds__(512)
streams_step_wide_kernel(const StreamsArgs a) {
  extern __shared__ float u_s[];                                     // [H rounded up to eight]
  __shared__ float scratch[32];
  __shared__ float mix_s[STREAMS_MAX * STREAMS_MAX], out_s[STREAMS_MAX], in_s[STREAMS_MAX];
  for (int i = threadIdx.x; i < STREAMS_MAX * STREAMS_MAX; i += blockDim.x) {
    const int to = i / STREAMS_MAX, from = i % STREAMS_MAX;
    mix_s[i] = to < a.S && from < a.S ? a.mix[from * a.S + to] : 0.f;
  }
  if (threadIdx.x < a.S) {
    out_s[threadIdx.x] = a.mult * a.out[threadIdx.x];
    in_s[threadIdx.x] = a.in != nullptr ? a.in[threadIdx.x] : 1.f;
  }
  __syncthreads();
  const T* yr = reinterpret_cast<const T*>(a.y);
  const T* w = reinterpret_cast<const T*>(a.w);
  T* xa = reinterpret_cast<T*>(a.xa);
  for (int t = blockIdx.x; t < a.rows; t += gridDim.x) {
    float ss[1] = {0.f};
    for (int i = threadIdx.x * 4; i < a.H; i += blockDim.x * 4) {    // (a row's pad holds zeros and may be read)
      float* x = a.x + t * a.ldx + i;
      float4 old[STREAMS_MAX];
#pragma unroll
      for (int s = 0; s < STREAMS_MAX; ++s)
        old[s] = s < a.S ? *reinterpret_cast<const float4*>(x + s * a.ldr) : make_float4(0.f, 0.f, 0.f, 0.f);
      float y[4], u[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int j = 0; j < 4; ++j) y[j] = i + j < a.H ? ld1(yr + t * a.ldy + i + j) : 0.f;
#pragma unroll 1
      for (int to = 0; to < a.S; ++to) {
        const float o = out_s[to], in = in_s[to];
        float4 v = make_float4(o * y[0], o * y[1], o * y[2], o * y[3]);
#pragma unroll
        for (int s = 0; s < STREAMS_MAX; ++s) {
          const float m = mix_s[to * STREAMS_MAX + s];
          v.x = fmaf(m, old[s].x, v.x);
          v.y = fmaf(m, old[s].y, v.y);
          v.z = fmaf(m, old[s].z, v.z);
          v.w = fmaf(m, old[s].w, v.w);
        }
        if (a.store) *reinterpret_cast<float4*>(x + to * a.lds) = v;
        u[0] = fmaf(in, v.x, u[0]);
        u[1] = fmaf(in, v.y, u[1]);
        u[2] = fmaf(in, v.z, u[2]);
        u[3] = fmaf(in, v.w, u[3]);
      }
      *reinterpret_cast<float4*>(u_s + i) = make_float4(u[0], u[1], u[2], u[3]);
#pragma unroll
      for (int j = 0; j < 4; ++j) ss[0] += u[j] * u[j];
    }
    block_sum<1>(ss, scratch);
    const float r = 1.f / sqrtf(ss[0] / static_cast<float>(a.H) + a.eps);
    for (int i = threadIdx.x * 4; i < a.H; i += blockDim.x * 4)      // each thread reads back what it wrote
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (i + j < a.H) st1(xa + t * a.lda + i + j, u_s[i + j] * r * (a.offset + ld1(w + i + j)));
  }
}

template <typename T, int VPT>
__global__ void __launch_bounds__(512)
embed_streams_kernel(const StreamsArgs a) {
  __shared__ float scratch[32];
  float in = 0.f;
  for (int s = 0; s < a.S; ++s) in += a.in != nullptr ? a.in[s] : 1.f;
  for (int t = blockIdx.x; t < a.rows; t += gridDim.x) {
    const int id = a.ids[t];
    const bool ok = id >= 0 && id < a.vocab;
    const T* src = reinterpret_cast<const T*>(a.table) + (ok ? id : 0) * a.ldt;
    float u[VPT][8], ss = 0.f;
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (threadIdx.x + k * blockDim.x) * 8, n = a.H - i;
#pragma unroll
      for (int j = 0; j < 8; ++j) u[k][j] = 0.f;
      if (n <= 0) continue;
      if (ok) ld8n<true>(src + i, n, u[k]);
      st8n<true>(a.x + t * a.ldx + i, n, u[k]);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        u[k][j] *= in;
        ss += u[k][j] * u[k][j];
      }
    }
    streams_norm<T, VPT>(a, t, u, ss, scratch);
  }
}

static bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename T, int VPT>
static void launch_streams(const StreamsArgs& a, int grid, int threads, cudaStream_t stream) {
  if (a.ids != nullptr) embed_streams_kernel<T, VPT><<<grid, threads, 0, stream>>>(a);
  else if (a.S <= 2) streams_step_kernel<T, VPT, 2><<<grid, threads, 0, stream>>>(a);
  else if (a.S <= 4) streams_step_kernel<T, VPT, 4><<<grid, threads, 0, stream>>>(a);
  else {
    const int smem = (a.H + 7) / 8 * 8 * 4;
    cudaFuncSetAttribute(streams_step_wide_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    streams_step_wide_kernel<T><<<grid, threads, smem, stream>>>(a);
  }
}

static int run_streams(const StreamsArgs& a, int dtype, const char* what, cudaStream_t stream) {
  const int nvec = (a.H + 7) / 8, vpt = nvec <= 512 ? 1 : nvec <= 1024 ? 2 : 4;
  const int threads = ((nvec + vpt - 1) / vpt + 31) / 32 * 32;
  if (a.H <= 0 || threads > 512 || a.S < 1 || a.S > STREAMS_MAX) {
    set_last_error("%s: %d streams of %d elements (up to %d streams of 16384)", what, a.S, a.H, STREAMS_MAX);
    return 1;
  }
  if (a.ldy % 8 != 0 || a.ldx % 8 != 0 || a.lds % 8 != 0 || a.lda % 8 != 0 || a.ldt % 8 != 0 || !aligned16(a.y) ||
      !aligned16(a.x) || !aligned16(a.w) || !aligned16(a.xa) || !aligned16(a.table) || a.lds < a.H) {
    set_last_error("%s: rows on 16-byte boundaries are needed", what);
    return 1;
  }
  const int cap = device_sm_count() * (threads <= 128 ? 16 : threads <= 256 ? 8 : 4);
  const int grid = a.rows < cap ? a.rows : cap;
#define TW_GO(TT)                                                      \
  do {                                                                 \
    if (vpt == 1) launch_streams<TT, 1>(a, grid, threads, stream);     \
    else if (vpt == 2) launch_streams<TT, 2>(a, grid, threads, stream); \
    else launch_streams<TT, 4>(a, grid, threads, stream);              \
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

extern "C" int tw_embed_streams(const int* ids, const void* table, long long ldt, int vocab, float* x, long long ldx,
                                long long lds, int S, const float* in, const void* w, float offset, void* xa, long long lda,
                                int T, int H, float eps, int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  StreamsArgs a{};
  a.x = x; a.ldx = ldx; a.lds = lds; a.in = in; a.w = w; a.offset = offset; a.xa = xa; a.lda = lda;
  a.rows = T; a.H = H; a.S = S; a.store = 1; a.eps = eps;
  a.ids = ids; a.table = table; a.ldt = ldt; a.vocab = vocab;
  return run_streams(a, dtype, "embed_streams", stream);
}

extern "C" int tw_streams_step(const void* y, long long ldy, float* x, long long ldx, long long lds, int S,
                               const float* mix, const float* out, float mult, const float* in, int first, int store,
                               const void* w, float offset, void* xa, long long lda, int T, int H, float eps, int dtype,
                               cudaStream_t stream) {
  if (T <= 0) return 0;
  StreamsArgs a{};
  a.y = y; a.ldy = ldy; a.x = x; a.ldx = ldx; a.lds = lds; a.mix = mix; a.out = out; a.in = in; a.mult = mult;
  a.w = w; a.offset = offset; a.xa = xa; a.lda = lda;
  a.rows = T; a.H = H; a.S = S; a.store = store; a.eps = eps;
  a.ldr = first ? 0 : lds;
  return run_streams(a, dtype, "streams_step", stream);
}
