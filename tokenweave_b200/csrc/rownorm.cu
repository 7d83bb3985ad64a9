// Row-wise kernels around the fp32 residual stream and the feed-forward of hybrid decoders.
// The residual stream is fp32; activations are bf16 or fp32 (template argument), all arithmetic is fp32.
//
//   tw_embed_residual   x32 = table[id] (the residual stream), xa = the same in the activation type
//   tw_postnorm_add     x32 += rmsnorm(y) * w ; xa = x32, or rmsnorm(x32) * w_final behind the last layer
//   tw_polynorm         out = a N(z) + b N(z^2) + c N(z^3) + e with N(v) = v / rms(v) over the row, powers
//                       element by element (the activation between the two matrices of a feed-forward)
//   tw_gated_group_norm out = groupnorm_rms(y * silu(z)) * w, the row cut in equal groups, each with its own
//                       root mean square (what follows a state-space recurrence)
//   tw_embed_norm       x32 = table[id] + pairs[row(previous id, id)] ; first = x32 ; xa = rmsnorm(x32) * w
//   tw_add_prenorm      x32 += y (+ first) ; xa = rmsnorm(x32) * w (the next layer's norm, or the final one)
//   tw_norm_gate        out = rmsnorm(y) * w * sigmoid(gate) * scale, the mean over `count` of the row's elements
//   tw_act_cols, tw_glu  activations behind a projection, for the fp32 products (the bf16 product has them in its
//                       epilogue): silu or relu^2 in place, act(z_gate) * z_up
//
// One CTA per row (per row and group), the row kept in registers between the passes when it fits.
#include "tw_host.h"
#include "tw_kernels.h"
#include "tw_typed.cuh"

namespace tw {

template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
embed_residual_kernel(const int* __restrict__ ids, const T* __restrict__ table, long long ldt, float* __restrict__ x32,
                      long long ldx, T* __restrict__ xa, long long lda, int H, int vocab) {
  const int t = blockIdx.x;
  const int id = ids[t];
  const bool ok = id >= 0 && id < vocab;
  const T* src = table + (ok ? id : 0) * ldt;
  for (int i = threadIdx.x * 8; i < H; i += blockDim.x * 8) {
    float v[8];
    ld8n<VEC>(src + i, H - i, v);
    if (!ok) {
#pragma unroll
      for (int j = 0; j < 8; ++j) v[j] = 0.f;
    }
    st8n<VEC>(x32 + t * ldx + i, H - i, v);
    st8n<VEC>(xa + t * lda + i, H - i, v);
  }
}

// VPT groups of eight elements per thread stay in registers.
template <typename T, bool VEC, int VPT>
__global__ void __launch_bounds__(1024)
postnorm_add_kernel(const T* __restrict__ y, long long ldy, float* __restrict__ x32, long long ldx,
                    const T* __restrict__ w, T* __restrict__ xa, long long lda, const T* __restrict__ w_final, int rows,
                    int H, float eps) {
  __shared__ float scratch[32];
  for (int t = blockIdx.x; t < rows; t += gridDim.x) {
    float v[VPT][8];
    float ss[1] = {0.f};
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (threadIdx.x + k * blockDim.x) * 8;
      ld8n<VEC>(y + t * ldy + i, H - i, v[k]);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss[0] += v[k][j] * v[k][j];
    }
    block_sum<1>(ss, scratch);
    const float r = 1.f / sqrtf(ss[0] / static_cast<float>(H) + eps);
    ss[0] = 0.f;
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (threadIdx.x + k * blockDim.x) * 8;
      if (i >= H) continue;
      float x[8], g[8];
      ld8n<VEC>(x32 + t * ldx + i, H - i, x);
      ld8n<VEC>(w + i, H - i, g);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        x[j] += v[k][j] * r * g[j];
        v[k][j] = x[j];
        ss[0] += x[j] * x[j];
      }
      st8n<VEC>(x32 + t * ldx + i, H - i, x);
      if (w_final == nullptr) st8n<VEC>(xa + t * lda + i, H - i, x);
    }
    if (w_final != nullptr) {
      block_sum<1>(ss, scratch);
      const float rf = 1.f / sqrtf(ss[0] / static_cast<float>(H) + eps);
#pragma unroll
      for (int k = 0; k < VPT; ++k) {
        const int i = (threadIdx.x + k * blockDim.x) * 8;
        if (i >= H) continue;
        float g[8], o[8];
        ld8n<VEC>(w_final + i, H - i, g);
#pragma unroll
        for (int j = 0; j < 8; ++j) o[j] = v[k][j] * rf * g[j];
        st8n<VEC>(xa + t * lda + i, H - i, o);
      }
    }
  }
}

template <typename T, bool VEC, int VPT>
__global__ void __launch_bounds__(1024)
polynorm_kernel(const T* __restrict__ z, long long ldz, const T* __restrict__ coef, T* __restrict__ out, long long ldo,
                int rows, int F, float eps) {
  __shared__ float scratch[96];
  const float ca = ld1(coef), cb = ld1(coef + 1), cc = ld1(coef + 2), ce = ld1(coef + 3);
  for (int t = blockIdx.x; t < rows; t += gridDim.x) {
    float v[VPT][8];
    float s[3] = {0.f, 0.f, 0.f};
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (threadIdx.x + k * blockDim.x) * 8;
      ld8n<VEC>(z + t * ldz + i, F - i, v[k]);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float q = v[k][j] * v[k][j];
        s[0] += q;
        s[1] += q * q;
        s[2] += q * q * q;
      }
    }
    block_sum<3>(s, scratch);
    const float n = static_cast<float>(F);
    const float ra = ca / sqrtf(s[0] / n + eps), rb = cb / sqrtf(s[1] / n + eps), rc = cc / sqrtf(s[2] / n + eps);
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (threadIdx.x + k * blockDim.x) * 8;
      if (i >= F) continue;
      float o[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float a = v[k][j];
        o[j] = ((rc * a + rb) * a + ra) * a + ce;
      }
      st8n<VEC>(out + t * ldo + i, F - i, o);
    }
  }
}

template <typename T, bool VEC, int VPT>
__global__ void __launch_bounds__(1024)
gated_group_norm_kernel(const T* __restrict__ y, long long ldy, const T* __restrict__ z, long long ldz,
                        const T* __restrict__ w, T* __restrict__ out, long long ldo, int items, int groups, int part,
                        float eps) {
  __shared__ float scratch[32];
  for (int it = blockIdx.x; it < items; it += gridDim.x) {
    const int t = it / groups, c0 = (it - t * groups) * part;
    float v[VPT][8];
    float ss[1] = {0.f};
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (threadIdx.x + k * blockDim.x) * 8;
      float g[8];
      ld8n<VEC>(y + t * ldy + c0 + i, part - i, v[k]);
      ld8n<VEC>(z + t * ldz + c0 + i, part - i, g);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        v[k][j] *= silu_t<T>(g[j]);
        ss[0] += v[k][j] * v[k][j];
      }
    }
    block_sum<1>(ss, scratch);
    const float r = 1.f / sqrtf(ss[0] / static_cast<float>(part) + eps);
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (threadIdx.x + k * blockDim.x) * 8;
      if (i >= part) continue;
      float g[8];
      ld8n<VEC>(w + c0 + i, part - i, g);
#pragma unroll
      for (int j = 0; j < 8; ++j) g[j] = v[k][j] * r * g[j];
      st8n<VEC>(out + t * ldo + c0 + i, part - i, g);
    }
  }
}

struct EmbedArgs {
  const int* ids;
  const void* table; long long ldt; int vocab;
  const void* pairs; long long ldp;                  // [buckets + 1, H]; null: no pair embeddings
  long long buckets, mul_prev, mul_cur;
  const int *row_seq, *cu_q, *prev_token;            // the token before a sequence's first row of the step, -1: none
  float* x32; long long ldx;
  float* first; long long ldf;                       // null: not kept
  const void* w;
  void* xa; long long lda;
  int rows, H;
  float eps;
};

template <typename T, bool VEC, int VPT>
__global__ void __launch_bounds__(1024)
embed_norm_kernel(const EmbedArgs a) {
  __shared__ float scratch[32];
  for (int t = blockIdx.x; t < a.rows; t += gridDim.x) {
    const int id = a.ids[t];
    const bool ok = id >= 0 && id < a.vocab;
    const T* src = reinterpret_cast<const T*>(a.table) + (ok ? id : 0) * a.ldt;
    const T* pair = nullptr;
    if (a.pairs != nullptr) {
      const int b = a.row_seq[t];
      const int prev = t == a.cu_q[b] ? a.prev_token[b] : a.ids[t - 1];
      long long row = a.buckets;
      if (prev >= 0) {
        row = (prev * a.mul_prev + id * a.mul_cur) % a.buckets;
        if (row < 0) row += a.buckets;
      }
      pair = reinterpret_cast<const T*>(a.pairs) + row * a.ldp;
    }
    float v[VPT][8];
    float ss[1] = {0.f};
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (threadIdx.x + k * blockDim.x) * 8;
      ld8n<VEC>(src + i, a.H - i, v[k]);
      if (!ok) {
#pragma unroll
        for (int j = 0; j < 8; ++j) v[k][j] = 0.f;
      }
      if (pair != nullptr) {
        float u[8];
        ld8n<VEC>(pair + i, a.H - i, u);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[k][j] += u[j];
      }
      if (i < a.H) {
        st8n<VEC>(a.x32 + t * a.ldx + i, a.H - i, v[k]);
        if (a.first != nullptr) st8n<VEC>(a.first + t * a.ldf + i, a.H - i, v[k]);
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) ss[0] += v[k][j] * v[k][j];
    }
    block_sum<1>(ss, scratch);
    const float r = 1.f / sqrtf(ss[0] / static_cast<float>(a.H) + a.eps);
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (threadIdx.x + k * blockDim.x) * 8;
      if (i >= a.H) continue;
      float g[8];
      ld8n<VEC>(reinterpret_cast<const T*>(a.w) + i, a.H - i, g);
#pragma unroll
      for (int j = 0; j < 8; ++j) g[j] = v[k][j] * r * g[j];
      st8n<VEC>(reinterpret_cast<T*>(a.xa) + t * a.lda + i, a.H - i, g);
    }
  }
}

template <typename T, bool VEC, int VPT>
__global__ void __launch_bounds__(1024)
add_prenorm_kernel(const T* __restrict__ y, long long ldy, float* __restrict__ x32, long long ldx,
                   const float* __restrict__ first, long long ldf, const T* __restrict__ w, T* __restrict__ xa,
                   long long lda, int rows, int H, float eps) {
  __shared__ float scratch[32];
  for (int t = blockIdx.x; t < rows; t += gridDim.x) {
    float v[VPT][8];
    float ss[1] = {0.f};
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (threadIdx.x + k * blockDim.x) * 8;
      float u[8];
      ld8n<VEC>(x32 + t * ldx + i, H - i, v[k]);
      ld8n<VEC>(y + t * ldy + i, H - i, u);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[k][j] += u[j];
      if (first != nullptr) {
        ld8n<VEC>(first + t * ldf + i, H - i, u);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[k][j] += u[j];
      }
      if (i < H) st8n<VEC>(x32 + t * ldx + i, H - i, v[k]);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss[0] += v[k][j] * v[k][j];
    }
    block_sum<1>(ss, scratch);
    const float r = 1.f / sqrtf(ss[0] / static_cast<float>(H) + eps);
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (threadIdx.x + k * blockDim.x) * 8;
      if (i >= H) continue;
      float g[8];
      ld8n<VEC>(w + i, H - i, g);
#pragma unroll
      for (int j = 0; j < 8; ++j) g[j] = v[k][j] * r * g[j];
      st8n<VEC>(xa + t * lda + i, H - i, g);
    }
  }
}

template <typename T, bool VEC, int VPT>
__global__ void __launch_bounds__(1024)
norm_gate_kernel(const T* __restrict__ y, long long ldy, const T* __restrict__ gate, long long ldg,
                 const T* __restrict__ w, T* __restrict__ out, long long ldo, int rows, int C, float count, float eps,
                 float scale) {
  __shared__ float scratch[32];
  for (int t = blockIdx.x; t < rows; t += gridDim.x) {
    float v[VPT][8];
    Raw8<T> graw[VPT];
    float ss[1] = {0.f};
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (threadIdx.x + k * blockDim.x) * 8;
      ld8n<VEC>(y + t * ldy + i, C - i, v[k]);
      graw[k] = ld8raw<VEC>(gate + t * ldg + i, C - i);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss[0] += v[k][j] * v[k][j];
    }
    block_sum<1>(ss, scratch);
    const float r = scale / sqrtf(ss[0] / count + eps);
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (threadIdx.x + k * blockDim.x) * 8;
      if (i >= C) continue;
      float g[8];
      ld8n<VEC>(w + i, C - i, g);
#pragma unroll
      for (int j = 0; j < 8; ++j) g[j] *= v[k][j] * r * sigmoid_t<T>(ld1(&graw[k].v[j]));
      st8n<VEC>(out + t * ldo + i, C - i, g);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
act_cols_kernel(T* __restrict__ x, long long ldx, int n, int act) {
  T* row = x + blockIdx.y * ldx;
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < n; i += gridDim.x * blockDim.x) {
    const float v = ld1(row + i), r = fmaxf(v, 0.f);
    st1(row + i, act == COL_RELU2 ? r * r : silu_t<T>(v));
  }
}

// z rows are [gate | up], d elements each; act: the kinds of the gated products
template <typename T>
__global__ void __launch_bounds__(256)
glu_kernel(const T* __restrict__ z, long long ldz, T* __restrict__ out, long long ldo, int d, int act, float limit,
           float alpha) {
  const T* row = z + blockIdx.y * ldz;
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < d; i += gridDim.x * blockDim.x) {
    float g = ld1(row + i), u = ld1(row + d + i);
    if (act == GLU_CLAMPED) {
      g = fminf(g, limit);
      u = fminf(fmaxf(u, -limit), limit) + 1.f;
      g *= sigmoid_t<T>(alpha * g);
    } else {
      g = act == GLU_GELU_TANH ? gelu_tanh_f(g) : silu_t<T>(g);
    }
    st1(out + blockIdx.y * ldo + i, g * u);
  }
}

static int check_launch(const char* what) {
  const cudaError_t e = cudaGetLastError();
  if (e == cudaSuccess) return 0;
  set_last_error("%s launch failed: %s", what, cudaGetErrorString(e));
  return 1;
}

// Threads and register groups for a row of n elements.
static bool row_shape(int n, int* threads, int* vpt, const char* what) {
  const int nvec = (n + 7) / 8;
  for (int v = 1; v <= 8; v *= 2) {
    const int th = ((nvec + v - 1) / v + 31) / 32 * 32;
    if (th <= 512 || (v == 8 && th <= 1024)) {
      *threads = th;
      *vpt = v;
      return true;
    }
  }
  set_last_error("%s: a row of %d elements is too long", what, n);
  return false;
}
static int row_grid(int items, int threads) {
  const int cap = device_sm_count() * (threads <= 128 ? 16 : threads <= 256 ? 8 : threads <= 512 ? 4 : 2);
  return items < cap ? items : cap;
}
static bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace tw

using namespace tw;

#define TW_ROW_VPT(KERNEL, T, VEC, ...)                                          \
  switch (vpt) {                                                                 \
    case 1: KERNEL<T, VEC, 1><<<grid, threads, 0, stream>>>(__VA_ARGS__); break; \
    case 2: KERNEL<T, VEC, 2><<<grid, threads, 0, stream>>>(__VA_ARGS__); break; \
    case 4: KERNEL<T, VEC, 4><<<grid, threads, 0, stream>>>(__VA_ARGS__); break; \
    default: KERNEL<T, VEC, 8><<<grid, threads, 0, stream>>>(__VA_ARGS__); break; \
  }

extern "C" int tw_embed_residual(const int* ids, const void* table, long long ldt, float* x32, long long ldx, void* xa,
                                 long long lda, int T, int H, int vocab, int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  const bool vec = ldt % 8 == 0 && ldx % 8 == 0 && lda % 8 == 0 && aligned16(table) && aligned16(x32) && aligned16(xa);
  int threads = ((H + 7) / 8 + 31) / 32 * 32;
  if (threads > 256) threads = 256;
#define TW_GO(TT, V)                                                                                       \
  embed_residual_kernel<TT, V><<<T, threads, 0, stream>>>(ids, reinterpret_cast<const TT*>(table), ldt, x32, ldx, \
                                                          reinterpret_cast<TT*>(xa), lda, H, vocab)
  if (dtype == TW_BF16) {
    if (vec) TW_GO(__nv_bfloat16, true); else TW_GO(__nv_bfloat16, false);
  } else {
    if (vec) TW_GO(float, true); else TW_GO(float, false);
  }
#undef TW_GO
  return check_launch("embed_residual");
}

extern "C" int tw_postnorm_add(const void* y, long long ldy, float* x32, long long ldx, const void* w, void* xa,
                               long long lda, const void* w_final, int T, int H, float eps, int dtype,
                               cudaStream_t stream) {
  if (T <= 0) return 0;
  int threads, vpt;
  if (!row_shape(H, &threads, &vpt, "postnorm_add")) return 1;
  const int grid = row_grid(T, threads);
  const bool vec = ldy % 8 == 0 && ldx % 8 == 0 && lda % 8 == 0 && aligned16(y) && aligned16(x32) && aligned16(xa) &&
                   aligned16(w) && aligned16(w_final);
#define TW_GO(TT, V)                                                                                              \
  TW_ROW_VPT(postnorm_add_kernel, TT, V, reinterpret_cast<const TT*>(y), ldy, x32, ldx,                           \
             reinterpret_cast<const TT*>(w), reinterpret_cast<TT*>(xa), lda, reinterpret_cast<const TT*>(w_final), \
             T, H, eps)
  if (dtype == TW_BF16) {
    if (vec) TW_GO(__nv_bfloat16, true) else TW_GO(__nv_bfloat16, false)
  } else {
    if (vec) TW_GO(float, true) else TW_GO(float, false)
  }
#undef TW_GO
  return check_launch("postnorm_add");
}

extern "C" int tw_polynorm(const void* z, long long ldz, const void* coef, void* out, long long ldo, int T, int F,
                           float eps, int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  int threads, vpt;
  if (!row_shape(F, &threads, &vpt, "polynorm")) return 1;
  const int grid = row_grid(T, threads);
  const bool vec = ldz % 8 == 0 && ldo % 8 == 0 && aligned16(z) && aligned16(out);
#define TW_GO(TT, V)                                                                                        \
  TW_ROW_VPT(polynorm_kernel, TT, V, reinterpret_cast<const TT*>(z), ldz, reinterpret_cast<const TT*>(coef), \
             reinterpret_cast<TT*>(out), ldo, T, F, eps)
  if (dtype == TW_BF16) {
    if (vec) TW_GO(__nv_bfloat16, true) else TW_GO(__nv_bfloat16, false)
  } else {
    if (vec) TW_GO(float, true) else TW_GO(float, false)
  }
#undef TW_GO
  return check_launch("polynorm");
}

extern "C" int tw_gated_group_norm(const void* y, long long ldy, const void* z, long long ldz, const void* w, void* out,
                                   long long ldo, int T, int C, int groups, float eps, int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (groups <= 0 || C % groups != 0) {
    set_last_error("gated_group_norm: %d channels do not divide into %d groups", C, groups);
    return 1;
  }
  const int part = C / groups;
  int threads, vpt;
  if (!row_shape(part, &threads, &vpt, "gated_group_norm")) return 1;
  const int grid = row_grid(T * groups, threads);
  const bool vec = ldy % 8 == 0 && ldz % 8 == 0 && ldo % 8 == 0 && (groups == 1 || part % 8 == 0) && aligned16(y) &&
                   aligned16(z) && aligned16(w) && aligned16(out);
#define TW_GO(TT, V)                                                                                                \
  TW_ROW_VPT(gated_group_norm_kernel, TT, V, reinterpret_cast<const TT*>(y), ldy, reinterpret_cast<const TT*>(z), ldz, \
             reinterpret_cast<const TT*>(w), reinterpret_cast<TT*>(out), ldo, T * groups, groups, part, eps)
  if (dtype == TW_BF16) {
    if (vec) TW_GO(__nv_bfloat16, true) else TW_GO(__nv_bfloat16, false)
  } else {
    if (vec) TW_GO(float, true) else TW_GO(float, false)
  }
#undef TW_GO
  return check_launch("gated_group_norm");
}

extern "C" int tw_embed_norm(const int* ids, const void* table, long long ldt, int vocab, const void* pairs, long long ldp,
                             long long buckets, long long mul_prev, long long mul_cur, const int* row_seq,
                             const int* cu_q, const int* prev_token, float* x32, long long ldx, float* first,
                             long long ldf, const void* w, void* xa, long long lda, int T, int H, float eps, int dtype,
                             cudaStream_t stream) {
  if (T <= 0) return 0;
  if (pairs != nullptr && (buckets <= 0 || row_seq == nullptr || prev_token == nullptr)) {
    set_last_error("embed_norm: token pairs need buckets and the tokens before the rows");
    return 1;
  }
  int threads, vpt;
  if (!row_shape(H, &threads, &vpt, "embed_norm")) return 1;
  const int grid = row_grid(T, threads);
  const bool vec = ldt % 8 == 0 && ldp % 8 == 0 && ldx % 8 == 0 && ldf % 8 == 0 && lda % 8 == 0 && aligned16(table) &&
                   aligned16(pairs) && aligned16(x32) && aligned16(first) && aligned16(w) && aligned16(xa);
  const EmbedArgs a{ids, table, ldt, vocab, pairs, ldp, buckets, mul_prev, mul_cur, row_seq, cu_q, prev_token,
                    x32, ldx, first, ldf, w, xa, lda, T, H, eps};
  if (dtype == TW_BF16) {
    if (vec) { TW_ROW_VPT(embed_norm_kernel, __nv_bfloat16, true, a) } else { TW_ROW_VPT(embed_norm_kernel, __nv_bfloat16, false, a) }
  } else {
    if (vec) { TW_ROW_VPT(embed_norm_kernel, float, true, a) } else { TW_ROW_VPT(embed_norm_kernel, float, false, a) }
  }
  return check_launch("embed_norm");
}

extern "C" int tw_add_prenorm(const void* y, long long ldy, float* x32, long long ldx, const float* first, long long ldf,
                              const void* w, void* xa, long long lda, int T, int H, float eps, int dtype,
                              cudaStream_t stream) {
  if (T <= 0) return 0;
  int threads, vpt;
  if (!row_shape(H, &threads, &vpt, "add_prenorm")) return 1;
  const int grid = row_grid(T, threads);
  const bool vec = ldy % 8 == 0 && ldx % 8 == 0 && ldf % 8 == 0 && lda % 8 == 0 && aligned16(y) && aligned16(x32) &&
                   aligned16(first) && aligned16(w) && aligned16(xa);
#define TW_GO(TT, V)                                                                                             \
  TW_ROW_VPT(add_prenorm_kernel, TT, V, reinterpret_cast<const TT*>(y), ldy, x32, ldx, first, ldf,               \
             reinterpret_cast<const TT*>(w), reinterpret_cast<TT*>(xa), lda, T, H, eps)
  if (dtype == TW_BF16) {
    if (vec) TW_GO(__nv_bfloat16, true) else TW_GO(__nv_bfloat16, false)
  } else {
    if (vec) TW_GO(float, true) else TW_GO(float, false)
  }
#undef TW_GO
  return check_launch("add_prenorm");
}

extern "C" int tw_norm_gate(const void* y, long long ldy, const void* gate, long long ldg, const void* w, void* out,
                            long long ldo, int T, int C, int count, float eps, float scale, int dtype,
                            cudaStream_t stream) {
  if (T <= 0) return 0;
  if (count <= 0 || count > C) {
    set_last_error("norm_gate: %d elements of a row of %d", count, C);
    return 1;
  }
  int threads, vpt;
  if (!row_shape(C, &threads, &vpt, "norm_gate")) return 1;
  const int grid = row_grid(T, threads);
  const bool vec = ldy % 8 == 0 && ldg % 8 == 0 && ldo % 8 == 0 && aligned16(y) && aligned16(gate) && aligned16(w) &&
                   aligned16(out);
#define TW_GO(TT, V)                                                                                                 \
  TW_ROW_VPT(norm_gate_kernel, TT, V, reinterpret_cast<const TT*>(y), ldy, reinterpret_cast<const TT*>(gate), ldg,   \
             reinterpret_cast<const TT*>(w), reinterpret_cast<TT*>(out), ldo, T, C, static_cast<float>(count), eps, scale)
  if (dtype == TW_BF16) {
    if (vec) TW_GO(__nv_bfloat16, true) else TW_GO(__nv_bfloat16, false)
  } else {
    if (vec) TW_GO(float, true) else TW_GO(float, false)
  }
#undef TW_GO
  return check_launch("norm_gate");
}

// Grid of the two elementwise kernels; the row is the second grid dimension, launched in blocks of 65535 rows.
extern "C" int tw_act_cols(void* x, long long ldx, int T, int n, int act, int dtype, cudaStream_t stream) {
  if (T <= 0 || n <= 0) return 0;
  if (act != COL_SILU && act != COL_RELU2) {
    set_last_error("act_cols: unknown activation %d", act);
    return 1;
  }
  const int gx = (n + 1023) / 1024;
  for (int t = 0; t < T; t += 65535) {
    const dim3 grid(gx, T - t < 65535 ? T - t : 65535);
    if (dtype == TW_BF16) act_cols_kernel<<<grid, 256, 0, stream>>>(reinterpret_cast<__nv_bfloat16*>(x) + t * ldx, ldx, n, act);
    else act_cols_kernel<<<grid, 256, 0, stream>>>(reinterpret_cast<float*>(x) + t * ldx, ldx, n, act);
  }
  return check_launch("act_cols");
}

extern "C" int tw_glu(const void* z, long long ldz, void* out, long long ldo, int T, int d, int act, float limit,
                      float alpha, int dtype, cudaStream_t stream) {
  if (T <= 0 || d <= 0) return 0;
  if (act < GLU_SILU || act > GLU_CLAMPED) {
    set_last_error("glu: unknown activation %d", act);
    return 1;
  }
  const int gx = (d + 1023) / 1024;
  for (int t = 0; t < T; t += 65535) {
    const dim3 grid(gx, T - t < 65535 ? T - t : 65535);
    if (dtype == TW_BF16)
      glu_kernel<<<grid, 256, 0, stream>>>(reinterpret_cast<const __nv_bfloat16*>(z) + t * ldz, ldz,
                                           reinterpret_cast<__nv_bfloat16*>(out) + t * ldo, ldo, d, act, limit, alpha);
    else
      glu_kernel<<<grid, 256, 0, stream>>>(reinterpret_cast<const float*>(z) + t * ldz, ldz,
                                           reinterpret_cast<float*>(out) + t * ldo, ldo, d, act, limit, alpha);
  }
  return check_launch("glu");
}
