// Latent attention (keys and values are linear maps of one low-rank latent per token): the kernels around the paged
// latent cache, for bf16 and fp32 storage and any sizes.
//
// A cache row holds [latent c (kv_rank) | zero pad | rotated key part (rot) | zero pad], both parts padded to eight
// elements, `row` elements in all. In the absorbed form a head's query for such a row is
// [W_uk^T q_unrotated | pad | q_rotated | pad] (W_uk: the head's key map), so a score is one dot product over a row,
// the value is the latent part of the same row, and the head's output is W_uv applied to the weighted latent sum.
//
//   tw_latent_prep     per token: RMS norm of the query latent; RMS norm of the key/value latent and rotation of the
//                      shared key part, both written straight into the cache slot
//   tw_rope_tail       rotates the tail of every head of q in place (the un-absorbed prefill form)
//   tw_latent_query    the rotated tail and the pads of absorbed query rows
//   tw_head_gemm       out[t, h, :] = B[h] a[t, h, :] for every head, rows through optional index lists, optionally
//                      times sigmoid(gate) element by element (tensor cores for bf16)
//   tw_latent_attn     absorbed causal attention of single query rows over the paged cache, fp32 softmax; sliding window,
//                      sink per head
//   tw_latent_gather   cache rows of some sequences, in order and from a given key on, into one contiguous buffer
#include "tw_host.h"
#include "tw_kernels.h"
#include "tw_mma.cuh"
#include "tw_typed.cuh"

namespace tw {

__device__ __forceinline__ int round8(int x) { return (x + 7) & ~7; }

// One CTA per token. The groups of eight of the query latent and of the key/value latent are dealt to the threads in one
// sequence and stay in registers between the sums and the writes.
template <typename T, bool VEC, int VPT>
__global__ void __launch_bounds__(256)
latent_prep_kernel(const T* __restrict__ p, long long ldp, int q_off, int q_rank, const T* __restrict__ wq,
                   T* __restrict__ cq, long long ldcq, int kv_off, int kv_rank, const T* __restrict__ wkv, int rot,
                   int rot_dims, const float* __restrict__ cos_sin, const int* __restrict__ positions,
                   const int* __restrict__ slots, T* __restrict__ cache, int row, float eps) {
  __shared__ float scratch[64];
  const int t = blockIdx.x;
  const T* src = p + t * ldp;
  const int nq = (q_rank + 7) >> 3, n_all = nq + ((kv_rank + 7) >> 3);
  float v[VPT][8], g[VPT][8];
  float s[2] = {0.f, 0.f};
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    const bool is_q = i < nq;
    const int c = (is_q ? i : i - nq) * 8, n = i < n_all ? (is_q ? q_rank : kv_rank) - c : 0;
    ld8n<VEC>(src + (is_q ? q_off : kv_off) + c, n, v[k]);
    ld8n<VEC>((is_q ? wq : wkv) + c, n, g[k]);
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += v[k][j] * v[k][j];
    if (is_q) s[0] += ss; else s[1] += ss;
  }
  block_sum<2>(s, scratch);
  const float rq = 1.f / sqrtf(s[0] / static_cast<float>(q_rank) + eps);
  const float rk = 1.f / sqrtf(s[1] / static_cast<float>(kv_rank) + eps);
  const int slot = slots[t];
  T* dst = cache + static_cast<long long>(slot < 0 ? 0 : slot) * row;
  const int rp = round8(kv_rank);
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i >= n_all) continue;
    const bool is_q = i < nq;
    const int c = (is_q ? i : i - nq) * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) v[k][j] = v[k][j] * (is_q ? rq : rk) * g[k][j];
    if (is_q) st8n<VEC>(cq + t * ldcq + c, q_rank - c, v[k]);
    else if (slot >= 0) st8(dst + c, v[k]);          // the pad behind the latent is written as zeros
  }
  if (slot < 0) return;
  const float* cs = cos_sin + static_cast<long long>(positions[t]) * rot_dims;
  const int half = rot_dims >> 1;
  for (int i = threadIdx.x; i < row - rp; i += blockDim.x) {
    float v = 0.f;
    if (i < half) {
      v = ld1(src + kv_off + kv_rank + i) * cs[i] - ld1(src + kv_off + kv_rank + half + i) * cs[half + i];
    } else if (i < rot_dims) {
      v = ld1(src + kv_off + kv_rank + i) * cs[i - half] + ld1(src + kv_off + kv_rank + i - half) * cs[i];
    } else if (i < rot) {
      v = ld1(src + kv_off + kv_rank + i);
    }
    st1(dst + rp + i, v);
  }
}

// Rotates elements [off, off + rot_dims) of every head of every row in place; VEC: eight pairs per thread.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
rope_tail_kernel(T* __restrict__ q, long long ldq, int heads, int head_stride, int off, int rot_dims,
                 const float* __restrict__ cos_sin, const int* __restrict__ positions) {
  const int t = blockIdx.x;
  const int half = rot_dims >> 1;
  const float* cs = cos_sin + static_cast<long long>(positions[t]) * rot_dims;
  constexpr int W = VEC ? 8 : 1;
  const int per = half / W;
  for (int i = threadIdx.x; i < heads * per; i += blockDim.x) {
    const int h = i / per, j = (i - h * per) * W;
    T* u = q + t * ldq + h * head_stride + off + j;
    if (VEC) {
      float a[8], b[8], c[8], s[8];
      ld8(u, a);
      ld8(u + half, b);
      ld8(cs + j, c);
      ld8(cs + half + j, s);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const float x = a[e] * c[e] - b[e] * s[e];
        b[e] = b[e] * c[e] + a[e] * s[e];
        a[e] = x;
      }
      st8(u, a);
      st8(u + half, b);
    } else {
      const float a = ld1(u), b = ld1(u + half), c = cs[j], s = cs[half + j];
      st1(u, a * c - b * s);
      st1(u + half, b * c + a * s);
    }
  }
}

// qa: [n, heads, row] absorbed queries; fills everything behind the kv_rank columns the head GEMM writes.
template <typename T>
__global__ void __launch_bounds__(256)
latent_query_kernel(const T* __restrict__ q, long long ldq, const int* __restrict__ rows, T* __restrict__ qa, int heads,
                    int head_stride, int off, int rot, int rot_dims, int kv_rank, int row,
                    const float* __restrict__ cos_sin, const int* __restrict__ positions) {
  const int i = blockIdx.x;
  const int t = rows[i];
  const int half = rot_dims >> 1;
  const int rp = round8(kv_rank), tail = row - kv_rank;
  const float* cs = cos_sin + static_cast<long long>(positions[t]) * rot_dims;
  for (int e = threadIdx.x; e < heads * tail; e += blockDim.x) {
    const int h = e / tail, c = kv_rank + e - h * tail, j = c - rp;
    const T* src = q + t * ldq + h * head_stride + off;
    float v = 0.f;
    if (j >= 0 && j < half) v = ld1(src + j) * cs[j] - ld1(src + half + j) * cs[half + j];
    else if (j >= half && j < rot_dims) v = ld1(src + j) * cs[j - half] + ld1(src + j - half) * cs[j];
    else if (j >= rot_dims && j < rot) v = ld1(src + j);
    st1(qa + (static_cast<long long>(i) * heads + h) * row + c, v);
  }
}

// ---- per-head matrix product -------------------------------------------------------------------------
struct HeadGemm {
  const void* A; long long lda; int a_hs; const int* a_rows;     // A[row, h * a_hs + k]
  const void* B; long long b_hs; int ldb;                        // B[h * b_hs + n * ldb + k]
  void* C; long long ldc; int c_hs; const int* c_rows;           // C[row, h * c_hs + n]
  const void* gate; long long ldg; int g_hs;                     // gate[c row, h * g_hs + n] or null
  int M, N, K;
};

constexpr int HG_M = 64, HG_N = 64, HG_K = 64;
constexpr int HG_LD = HG_K + 8;        // padded rows: conflict-free ldmatrix

constexpr int HG_STAGES = 4;
constexpr int HG_SMEM = HG_STAGES * (HG_M + HG_N) * HG_LD * 2;

// Eight elements of one row into shared memory, zeros behind the row's end and for rows outside the problem. VEC: K, the
// strides and the bases keep 16-byte groups aligned, the copy is asynchronous.
template <bool VEC>
__device__ __forceinline__ void hg_load(__nv_bfloat16* dst, const __nv_bfloat16* row, int k, int K, const void* base) {
  const bool ok = row != nullptr && k < K;
  if (VEC) {
    cp_async16(dst, ok ? static_cast<const void*>(row + k) : base, ok ? 16 : 0);    // zero bytes: base is not read
  } else {
    uint4 u = make_uint4(0, 0, 0, 0);
    __nv_bfloat16* e = reinterpret_cast<__nv_bfloat16*>(&u);
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (ok && k + j < K) e[j] = row[k + j];
    *reinterpret_cast<uint4*>(dst) = u;
  }
}

template <bool VEC>
__global__ void __launch_bounds__(128)
head_gemm_bf16_kernel(const HeadGemm g) {
  extern __shared__ __align__(16) __nv_bfloat16 hg_smem[];
  const int h = blockIdx.z, m0 = blockIdx.y * HG_M, n0 = blockIdx.x * HG_N;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int wm = (warp & 1) * 32, wn = (warp >> 1) * 32;
  const __nv_bfloat16* A = reinterpret_cast<const __nv_bfloat16*>(g.A) + static_cast<long long>(h) * g.a_hs;
  const __nv_bfloat16* B = reinterpret_cast<const __nv_bfloat16*>(g.B) + h * g.b_hs;
  float acc[2][4][4] = {};
  const int lr = threadIdx.x >> 3, lc = (threadIdx.x & 7) * 8;      // 16 rows x 8 groups per pass
  const __nv_bfloat16* arow[4];
  const __nv_bfloat16* brow[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + lr + 16 * i, n = n0 + lr + 16 * i;
    arow[i] = m < g.M ? A + (g.a_rows != nullptr ? g.a_rows[m] : m) * g.lda : nullptr;
    brow[i] = n < g.N ? B + static_cast<long long>(n) * g.ldb : nullptr;
  }
  const int steps = (g.K + HG_K - 1) / HG_K;
  auto load = [&](int step) {
    __nv_bfloat16* sa = hg_smem + (step % HG_STAGES) * (HG_M + HG_N) * HG_LD;
    if (step < steps) {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int off = (lr + 16 * i) * HG_LD + lc;
        hg_load<VEC>(sa + off, arow[i], step * HG_K + lc, g.K, g.A);
        hg_load<VEC>(sa + HG_M * HG_LD + off, brow[i], step * HG_K + lc, g.K, g.A);
      }
    }
    cp_async_commit();           // one group per step, empty behind the last
  };
#pragma unroll
  for (int i = 0; i < HG_STAGES - 1; ++i) load(i);
  for (int step = 0; step < steps; ++step) {
    cp_async_wait<HG_STAGES - 2>();
    __syncthreads();             // this step's tiles have landed, and everyone is done with the previous step's
    load(step + HG_STAGES - 1);
    const __nv_bfloat16* sa = hg_smem + (step % HG_STAGES) * (HG_M + HG_N) * HG_LD;
    const __nv_bfloat16* sb = sa + HG_M * HG_LD;
#pragma unroll
    for (int k = 0; k < HG_K; k += 16) {
      uint32_t a[2][4], b[2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        ldmatrix_x4(a[i], smem_u32(sa + (wm + i * 16) * HG_LD + k + frag_a(lane, HG_LD)));
        ldmatrix_x4(b[i], smem_u32(sb + (wn + i * 16) * HG_LD + k + frag_b(lane, HG_LD)));
      }
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) mma_bf16(acc[i][j], a[i], b[j >> 1][(j & 1) * 2], b[j >> 1][(j & 1) * 2 + 1]);
    }
  }
  __nv_bfloat16* C = reinterpret_cast<__nv_bfloat16*>(g.C) + static_cast<long long>(h) * g.c_hs;
  const __nv_bfloat16* gate = reinterpret_cast<const __nv_bfloat16*>(g.gate);
  // column pairs as one 4-byte access when every row starts on one
  const bool pairs = ((g.N | g.ldc | g.c_hs | g.ldg | g.g_hs) & 1) == 0 &&
                     ((reinterpret_cast<uintptr_t>(g.C) | reinterpret_cast<uintptr_t>(g.gate)) & 3) == 0;
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int m = m0 + wm + i * 16 + half * 8 + (lane >> 2);
      if (m >= g.M) continue;
      const long long r = g.c_rows != nullptr ? g.c_rows[m] : m;
      const __nv_bfloat16* grow = gate + r * g.ldg + static_cast<long long>(h) * g.g_hs;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int n = n0 + wn + j * 8 + (lane & 3) * 2;
        if (n >= g.N) continue;
        float2 v = make_float2(acc[i][j][half * 2], acc[i][j][half * 2 + 1]);
        if (pairs) {
          if (gate != nullptr) {
            const float2 s = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(grow + n));
            v.x *= sigmoid_t<__nv_bfloat16>(s.x);
            v.y *= sigmoid_t<__nv_bfloat16>(s.y);
          }
          *reinterpret_cast<uint32_t*>(C + r * g.ldc + n) = pack_bf16x2(v.x, v.y);
        } else {
          if (gate != nullptr) {
            v.x *= sigmoid_t<__nv_bfloat16>(ld1(grow + n));
            if (n + 1 < g.N) v.y *= sigmoid_t<__nv_bfloat16>(ld1(grow + n + 1));
          }
          st1(C + r * g.ldc + n, v.x);
          if (n + 1 < g.N) st1(C + r * g.ldc + n + 1, v.y);
        }
      }
    }
}

__global__ void __launch_bounds__(256)
head_gemm_f32_kernel(const HeadGemm g) {
  __shared__ float sa[16][64 + 4], sb[16][64 + 4];
  const int h = blockIdx.z, m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const float* A = reinterpret_cast<const float*>(g.A) + static_cast<long long>(h) * g.a_hs;
  const float* B = reinterpret_cast<const float*>(g.B) + h * g.b_hs;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < g.K; k0 += 16) {
    for (int i = threadIdx.x; i < 64 * 16; i += 256) {
      const int r = i >> 4, k = i & 15, m = m0 + r, n = n0 + r;
      const bool kin = k0 + k < g.K;
      sa[k][r] = (kin && m < g.M) ? A[(g.a_rows != nullptr ? g.a_rows[m] : m) * g.lda + k0 + k] : 0.f;
      sb[k][r] = (kin && n < g.N) ? B[static_cast<long long>(n) * g.ldb + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k)
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(sa[k][ty * 4 + i], sb[k][tx * 4 + j], acc[i][j]);
    __syncthreads();
  }
  float* C = reinterpret_cast<float*>(g.C) + static_cast<long long>(h) * g.c_hs;
  const float* gate = reinterpret_cast<const float*>(g.gate);
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= g.M) continue;
    const long long r = g.c_rows != nullptr ? g.c_rows[m] : m;
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= g.N) continue;
      float v = acc[i][j];
      if (gate != nullptr) v *= sigmoid_f(gate[r * g.ldg + static_cast<long long>(h) * g.g_hs + n]);
      C[r * g.ldc + n] = v;
    }
  }
}

// ---- absorbed attention, any sizes ---------------------------------------------------------------------
// One warp per (query row, head): lane l holds elements l, l + 32, ... of the query and of the output latent. A key
// costs one pass over its cache row: dot product, shuffle reduction, and the same registers feed the weighted sum.
template <typename T, int NK>
__global__ void __launch_bounds__(128)
latent_attn_kernel(const T* __restrict__ qa, const T* __restrict__ cache, const int* __restrict__ tok_seq,
                   const int* __restrict__ tok_kvlen, const int* __restrict__ block_table, int max_blocks, int page,
                   T* __restrict__ out, int heads, int row, int kv_rank, float scale, int window,
                   const float* __restrict__ sink) {
  const int i = blockIdx.x, h = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= heads) return;
  const long long item = static_cast<long long>(i) * heads + h;
  float q[NK], o[NK];
#pragma unroll
  for (int k = 0; k < NK; ++k) {
    const int c = lane + 32 * k;
    q[k] = c < row ? ld1(qa + item * row + c) * scale : 0.f;
    o[k] = 0.f;
  }
  const int* table = block_table + static_cast<long long>(tok_seq[i]) * max_blocks;
  const int n_keys = tok_kvlen[i];
  float m = -INFINITY, l = 0.f;
  for (int j0 = window > 0 ? max(0, n_keys - window) : 0; j0 < n_keys; j0 += 2) {
    float x[2][NK], s[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int j = min(j0 + u, n_keys - 1);
      const T* src = cache + (static_cast<long long>(table[j / page]) * page + j % page) * row;
      s[u] = 0.f;
#pragma unroll
      for (int k = 0; k < NK; ++k) {
        const int c = lane + 32 * k;
        x[u][k] = c < row ? ld1(src + c) : 0.f;
        s[u] = fmaf(q[k], x[u][k], s[u]);
      }
    }
#pragma unroll
    for (int u = 0; u < 2; ++u) s[u] = warp_sum(s[u]);
    if (j0 + 1 >= n_keys) s[1] = -INFINITY;
    const float mn = fmaxf(m, fmaxf(s[0], s[1]));
    const float a = expf(m - mn), p0 = expf(s[0] - mn), p1 = expf(s[1] - mn);
    m = mn;
    l = l * a + p0 + p1;
#pragma unroll
    for (int k = 0; k < NK; ++k) o[k] = fmaf(o[k], a, fmaf(p0, x[0][k], p1 * x[1][k]));
  }
  if (sink != nullptr) l += expf(sink[h] - m);
  const float inv = 1.f / l;
#pragma unroll
  for (int k = 0; k < NK; ++k) {
    const int c = lane + 32 * k;
    if (c < kv_rank) st1(out + item * kv_rank + c, o[k] * inv);
  }
}

constexpr int LG_ROWS = 16;      // rows per CTA

__global__ void __launch_bounds__(256)
latent_gather_kernel(const uint4* __restrict__ cache, uint4* __restrict__ dst, const int* __restrict__ seqs,
                     const int* __restrict__ cu, const int* __restrict__ from, const int* __restrict__ block_table,
                     int max_blocks, int page, int row_vec) {
  const int b = blockIdx.y;
  const int key0 = from != nullptr ? from[b] : 0;
  const int n = cu[b + 1] - cu[b], first = blockIdx.x * LG_ROWS;
  if (first >= n) return;
  const int* table = block_table + static_cast<long long>(seqs[b]) * max_blocks;
  const int items = min(LG_ROWS, n - first) * row_vec;
  for (int i = threadIdx.x; i < items; i += blockDim.x) {
    const int r = i / row_vec, v = i - r * row_vec, j = key0 + first + r;
    dst[(static_cast<long long>(cu[b]) + first + r) * row_vec + v] =
        cache[(static_cast<long long>(table[j / page]) * page + j % page) * row_vec + v];
  }
}

static int check_launch(const char* what) {
  const cudaError_t e = cudaGetLastError();
  if (e == cudaSuccess) return 0;
  set_last_error("%s launch failed: %s", what, cudaGetErrorString(e));
  return 1;
}
static bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace tw

using namespace tw;

extern "C" int tw_latent_prep(const void* p, long long ldp, int q_off, int q_rank, const void* wq, void* cq,
                              long long ldcq, int kv_off, int kv_rank, const void* wkv, int rot, int rot_dims,
                              const float* cos_sin, const int* positions, const int* slots, void* cache, int row, int T,
                              float eps, int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (row % 8 != 0 || rot_dims % 2 != 0 || rot_dims > rot || row < ((kv_rank + 7) & ~7) + rot) {
    set_last_error("latent_prep: bad row layout (row=%d, kv_rank=%d, rot=%d, rotated=%d)", row, kv_rank, rot, rot_dims);
    return 1;
  }
  const bool vec = ldp % 8 == 0 && q_off % 8 == 0 && kv_off % 8 == 0 && ldcq % 8 == 0 && aligned16(p) && aligned16(cq) &&
                   aligned16(wq) && aligned16(wkv);
  const int groups = (q_rank + 7) / 8 + (kv_rank + 7) / 8;
  const int threads = groups >= 256 ? 256 : (groups + 31) / 32 * 32;
  const int vpt = (groups + threads - 1) / threads;
#define TW_PREP(TT, V, N)                                                                                              \
  latent_prep_kernel<TT, V, N><<<T, threads, 0, stream>>>(                                                             \
      reinterpret_cast<const TT*>(p), ldp, q_off, q_rank, reinterpret_cast<const TT*>(wq), reinterpret_cast<TT*>(cq), \
      ldcq, kv_off, kv_rank, reinterpret_cast<const TT*>(wkv), rot, rot_dims, cos_sin, positions, slots,               \
      reinterpret_cast<TT*>(cache), row, eps)
#define TW_GO(TT, V)                       \
  do {                                     \
    if (vpt <= 1) TW_PREP(TT, V, 1);       \
    else if (vpt <= 2) TW_PREP(TT, V, 2);  \
    else if (vpt <= 4) TW_PREP(TT, V, 4);  \
    else TW_PREP(TT, V, 8);                \
  } while (0)
  if (vpt > 8) {
    set_last_error("latent_prep: latents of %d and %d elements are too long", q_rank, kv_rank);
    return 1;
  }
  if (dtype == TW_BF16) {
    if (vec) TW_GO(__nv_bfloat16, true); else TW_GO(__nv_bfloat16, false);
  } else {
    if (vec) TW_GO(float, true); else TW_GO(float, false);
  }
#undef TW_GO
#undef TW_PREP
  return check_launch("latent_prep");
}

extern "C" int tw_rope_tail(void* q, long long ldq, int T, int heads, int head_stride, int off, int rot_dims,
                            const float* cos_sin, const int* positions, int dtype, cudaStream_t stream) {
  if (T <= 0 || rot_dims <= 0) return 0;
  const bool vec = rot_dims % 16 == 0 && head_stride % 8 == 0 && off % 8 == 0 && ldq % 8 == 0 && aligned16(q) && aligned16(cos_sin);
  const int items = heads * (rot_dims / 2) / (vec ? 8 : 1);
  const int threads = items >= 256 ? 256 : (items + 31) / 32 * 32;
#define TW_GO(TT, V)                                                                                               \
  rope_tail_kernel<TT, V><<<T, threads, 0, stream>>>(reinterpret_cast<TT*>(q), ldq, heads, head_stride, off, rot_dims, \
                                                     cos_sin, positions)
  if (dtype == TW_BF16) {
    if (vec) TW_GO(__nv_bfloat16, true); else TW_GO(__nv_bfloat16, false);
  } else {
    if (vec) TW_GO(float, true); else TW_GO(float, false);
  }
#undef TW_GO
  return check_launch("rope_tail");
}

extern "C" int tw_latent_query(const void* q, long long ldq, const int* rows, int n, void* qa, int heads,
                               int head_stride, int off, int rot, int rot_dims, int kv_rank, int row,
                               const float* cos_sin, const int* positions, int dtype, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (dtype == TW_BF16)
    latent_query_kernel<__nv_bfloat16><<<n, 256, 0, stream>>>(
        reinterpret_cast<const __nv_bfloat16*>(q), ldq, rows, reinterpret_cast<__nv_bfloat16*>(qa), heads, head_stride,
        off, rot, rot_dims, kv_rank, row, cos_sin, positions);
  else
    latent_query_kernel<float><<<n, 256, 0, stream>>>(reinterpret_cast<const float*>(q), ldq, rows,
                                                      reinterpret_cast<float*>(qa), heads, head_stride, off, rot,
                                                      rot_dims, kv_rank, row, cos_sin, positions);
  return check_launch("latent_query");
}

extern "C" int tw_head_gemm(const void* A, long long lda, int a_hs, const int* a_rows, const void* B, long long b_hs,
                            int ldb, void* C, long long ldc, int c_hs, const int* c_rows, const void* gate,
                            long long ldg, int g_hs, int heads, int M, int N, int K, int dtype, cudaStream_t stream) {
  if (M <= 0 || N <= 0 || heads <= 0) return 0;
  const HeadGemm g{A, lda, a_hs, a_rows, B, b_hs, ldb, C, ldc, c_hs, c_rows, gate, ldg, g_hs, M, N, K};
  const dim3 grid((N + 63) / 64, (M + 63) / 64, heads);
  if (grid.y > 65535 || grid.z > 65535) {
    set_last_error("head_gemm: too many rows (%d) or heads (%d)", M, heads);
    return 1;
  }
  if (dtype == TW_BF16) {
    const bool vec = K % 8 == 0 && lda % 8 == 0 && a_hs % 8 == 0 && b_hs % 8 == 0 && ldb % 8 == 0 && aligned16(A) &&
                     aligned16(B);
    static thread_local int configured_dev = -1;
    int dev = 0;
    cudaGetDevice(&dev);
    if (configured_dev != dev) {
      cudaError_t e = cudaFuncSetAttribute(head_gemm_bf16_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, HG_SMEM);
      if (e == cudaSuccess)
        e = cudaFuncSetAttribute(head_gemm_bf16_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, HG_SMEM);
      if (e != cudaSuccess) {
        set_last_error("head_gemm: cudaFuncSetAttribute failed: %s", cudaGetErrorString(e));
        return 1;
      }
      configured_dev = dev;
    }
    if (vec) head_gemm_bf16_kernel<true><<<grid, 128, HG_SMEM, stream>>>(g);
    else head_gemm_bf16_kernel<false><<<grid, 128, HG_SMEM, stream>>>(g);
  } else {
    head_gemm_f32_kernel<<<grid, 256, 0, stream>>>(g);
  }
  return check_launch("head_gemm");
}

extern "C" int tw_latent_attn(const void* qa, const void* cache, const int* tok_seq, const int* tok_kvlen, int n,
                              const int* block_table, int max_blocks, int page, void* out, int heads, int row,
                              int kv_rank, float scale, int window, const float* sink, int dtype, cudaStream_t stream) {
  if (n <= 0) return 0;
  const dim3 grid(n, (heads + 3) / 4);
#define TW_GO(NK)                                                                                                      \
  do {                                                                                                                 \
    if (dtype == TW_BF16)                                                                                              \
      latent_attn_kernel<__nv_bfloat16, NK><<<grid, 128, 0, stream>>>(                                                 \
          reinterpret_cast<const __nv_bfloat16*>(qa), reinterpret_cast<const __nv_bfloat16*>(cache), tok_seq, tok_kvlen, \
          block_table, max_blocks, page, reinterpret_cast<__nv_bfloat16*>(out), heads, row, kv_rank, scale, window,    \
          sink);                                                                                                       \
    else                                                                                                               \
      latent_attn_kernel<float, NK><<<grid, 128, 0, stream>>>(                                                         \
          reinterpret_cast<const float*>(qa), reinterpret_cast<const float*>(cache), tok_seq, tok_kvlen, block_table,  \
          max_blocks, page, reinterpret_cast<float*>(out), heads, row, kv_rank, scale, window, sink);                  \
  } while (0)
  if (row <= 64) TW_GO(2);
  else if (row <= 128) TW_GO(4);
  else if (row <= 192) TW_GO(6);
  else if (row <= 320) TW_GO(10);
  else if (row <= 576) TW_GO(18);
  else if (row <= 1152) TW_GO(36);
  else {
    set_last_error("latent_attn: cache rows of up to 1152 elements are supported (got %d)", row);
    return 1;
  }
#undef TW_GO
  return check_launch("latent_attn");
}

extern "C" int tw_latent_gather(const void* cache, void* dst, const int* seqs, const int* cu, const int* from, int n_seqs,
                                int max_rows, const int* block_table, int max_blocks, int page, int row_bytes,
                                cudaStream_t stream) {
  if (n_seqs <= 0 || max_rows <= 0) return 0;
  if (row_bytes % 16 != 0) {
    set_last_error("latent_gather: rows of %d bytes are not a multiple of 16", row_bytes);
    return 1;
  }
  const dim3 grid((max_rows + LG_ROWS - 1) / LG_ROWS, n_seqs);
  latent_gather_kernel<<<grid, 256, 0, stream>>>(reinterpret_cast<const uint4*>(cache), reinterpret_cast<uint4*>(dst),
                                                 seqs, cu, from, block_table, max_blocks, page, row_bytes / 16);
  return check_launch("latent_gather");
}
