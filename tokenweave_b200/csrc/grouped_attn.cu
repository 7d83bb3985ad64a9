// Grouped-query attention with its own sizes of queries / keys and values, bf16 and fp32, any sizes.
//
//   tw_qkv_prep    everything between the projection and the attention in one pass over the projection's rows: causal
//                  convolution over time (with the sequence's kept inputs), RMS norm of queries and keys per head or over
//                  the whole projection (with weights, or per head without), rotation of the leading dimensions of
//                  queries and keys (neighbouring dimensions are a pair), query temperature, queries to a buffer, keys and
//                  values into the paged caches (no key heads: queries only).
//                  A step of single-token sequences moves the convolution's state on in the same launch
//   tw_attn_rows   attention of single query rows on SIMT: fp32, and heads beyond what the tensor-core kernels take
//                  (attn_prefill_split.cu, attn_decode_tc.cu); softmax with distance bias, sink, factor on the result,
//                  sliding window with kept first keys, or sigmoid weights with a bias per head, chunks and a gate
//
// Heads are padded to eight elements in the projection's rows, the query buffer and the caches; pads are zeros. All
// arithmetic is fp32.
#include "tw_host.h"
#include "tw_kernels.h"
#include "tw_typed.cuh"

namespace tw {

struct PrepArgs {
  const void* p; long long ldp;             // [T, heads * dp | kv_heads * dp | kv_heads * vp]
  int T, heads, kv_heads, dim, dp, vp;
  void* q; long long ldq;                   // [T, heads * dp]
  void *k_cache, *v_cache;                  // [slots of the cache, kv_heads, dp or vp]
  const int *positions, *cache_slots;
  const void* conv_w;                       // [taps, channels] (last tap = current token); null: none
  void* conv_state; int taps;               // [slots, taps - 1, channels], oldest first
  const int *row_seq, *cu_q, *kv_lens, *slots;
  int single;                               // one row per sequence: the state is moved on here
  const void *wq, *wk;                      // norm weights: [dp] each, or [heads * dp] and [kv_heads * dp]; null: ones
  float eps, temp_coef;
  int temp_every;
  const float* cos_sin; int rot_dims;       // [positions, rot_dims]: cosines, then sines, of the pairs; null: no rotation
};

// Eight channels from column c on of row t behind the convolution. UPDATE: also writes the state that follows the row
// (entries are read before they are written, each by the thread that owns the channels).
template <typename T, bool CONV, bool UPDATE>
__device__ __forceinline__ void prep_load(const PrepArgs& a, int t, int b, int start, bool past, int channels, int c,
                                          float (&y)[8]) {
  const T* p = reinterpret_cast<const T*>(a.p);
  if (!CONV) {
    ld8(p + t * a.ldp + c, y);
    return;
  }
#pragma unroll
  for (int j = 0; j < 8; ++j) y[j] = 0.f;
  T* st = reinterpret_cast<T*>(a.conv_state);
  if (a.taps > 1) st += static_cast<long long>(a.slots[b]) * (a.taps - 1) * channels + c;
  for (int k = 0; k < a.taps; ++k) {
    const int r = t - (a.taps - 1 - k);
    float u[8], w[8];
    if (r >= start) {
      ld8(p + r * a.ldp + c, u);
    } else if (past) {
      ld8(st + static_cast<long long>(a.taps - 1 - (start - r)) * channels, u);
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) u[j] = 0.f;
    }
    ld8(reinterpret_cast<const T*>(a.conv_w) + static_cast<long long>(k) * channels + c, w);
#pragma unroll
    for (int j = 0; j < 8; ++j) y[j] = fmaf(w[j], u[j], y[j]);
    // one row per sequence: entry k - 1 of the new state is this input, and entry k - 1 of the old one has been read
    if (UPDATE && k > 0) st8(st + static_cast<long long>(k - 1) * channels, u);
  }
}

__device__ __forceinline__ float query_temperature(const PrepArgs& a, int t) {
  return 1.f + a.temp_coef * logf(static_cast<float>((a.positions[t] + 1) / a.temp_every) + 1.f);
}

// Rotates the pairs among dimensions d .. d + 7 of a head whose first `dims` dimensions turn.
__device__ __forceinline__ void rotate_pairs(float (&v)[8], int d, int dims, const float* cs) {
  const int half = dims >> 1;
  float c[4], s[4];
  if ((half & 3) == 0) {
    if (d >= dims) return;
    *reinterpret_cast<float4*>(c) = *reinterpret_cast<const float4*>(cs + (d >> 1));
    *reinterpret_cast<float4*>(s) = *reinterpret_cast<const float4*>(cs + half + (d >> 1));
  } else {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const bool in = d + 2 * j < dims;
      c[j] = in ? cs[(d >> 1) + j] : 1.f;
      s[j] = in ? cs[half + (d >> 1) + j] : 0.f;
    }
  }
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float x = v[2 * j], y = v[2 * j + 1];
    v[2 * j] = x * c[j] - y * s[j];
    v[2 * j + 1] = y * c[j] + x * s[j];
  }
}

// One CTA per row; a group of S lanes (a power of two) takes one head at a time. NORM: 0 none, 1 per head, 2 whole.
template <typename T, int NORM, bool CONV, int S>
__global__ void __launch_bounds__(256)
qkv_prep_kernel(const PrepArgs a) {
  __shared__ float scratch[64];
  const int t = blockIdx.x;
  const int H = a.heads, G = a.kv_heads, nq = H * a.dp, nk = G * a.dp, channels = nq + nk + G * a.vp;
  const int sub = threadIdx.x & (S - 1), first = threadIdx.x / S, step = blockDim.x / S;
  int b = 0, start = 0;
  bool past = false;
  if (CONV) {
    b = a.row_seq[t];
    start = a.cu_q[b];
    past = a.kv_lens[b] > a.cu_q[b + 1] - start;
  }
  float whole[2] = {0.f, 0.f};
  if (NORM == 2) {
    for (int i = threadIdx.x * 8; i < nq + nk; i += blockDim.x * 8) {
      float v[8];
      prep_load<T, CONV, false>(a, t, b, start, past, channels, i, v);
      float s = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) s += v[j] * v[j];
      if (i < nq) whole[0] += s;
      else whole[1] += s;
    }
    block_sum<2>(whole, scratch);
    whole[0] = 1.f / sqrtf(whole[0] / static_cast<float>(H * a.dim) + a.eps);
    whole[1] = 1.f / sqrtf(whole[1] / static_cast<float>(G * a.dim) + a.eps);
  }
  const float temp = a.temp_coef != 0.f ? query_temperature(a, t) : 1.f;
  const float* cs = a.cos_sin != nullptr ? a.cos_sin + static_cast<long long>(a.positions[t]) * a.rot_dims : nullptr;
  const int slot = a.cache_slots[t];
  T* q = reinterpret_cast<T*>(a.q) + t * a.ldq;
  T* kc = reinterpret_cast<T*>(a.k_cache) + static_cast<long long>(slot) * nk;
  T* vc = reinterpret_cast<T*>(a.v_cache) + static_cast<long long>(slot) * G * a.vp;
  // whole warps stay in the loop: the lanes of a head that is not there add nothing to the shuffles below
  for (int h0 = 0; h0 < H + 2 * G; h0 += step) {
    const int h = h0 + first;
    const bool there = h < H + 2 * G;
    const bool is_v = h >= H + G;
    const int width = is_v ? a.vp : a.dp;
    const int base = is_v ? nq + nk + (h - H - G) * a.vp : h * a.dp;
    const bool normed = NORM != 0 && there && !is_v;
    const bool single = CONV && a.single;
    float r = 1.f, v[8];
    const int d0 = sub * 8;
    const bool mine = there && d0 < width;
    if (NORM == 1) {
      float s = 0.f;
      if (normed) {
        for (int d = d0; d < width; d += S * 8) {
          prep_load<T, CONV, false>(a, t, b, start, past, channels, base + d, v);
#pragma unroll
          for (int j = 0; j < 8; ++j) s += v[j] * v[j];
        }
      }
#pragma unroll
      for (int o = S / 2; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
      if (normed) r = 1.f / sqrtf(s / static_cast<float>(a.dim) + a.eps);
    } else if (NORM == 2) {
      r = h < H ? whole[0] : whole[1];
    }
    if (!mine) continue;
    const float f = h < H ? r * temp : r;
    for (int d = d0; d < width; d += S * 8) {
      if (single) prep_load<T, CONV, true>(a, t, b, start, past, channels, base + d, v);
      else prep_load<T, CONV, false>(a, t, b, start, past, channels, base + d, v);
      if (normed && a.wq == nullptr) {
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] *= f;
      } else if (normed) {
        float w[8];
        const T* wp = reinterpret_cast<const T*>(h < H ? a.wq : a.wk);
        ld8(wp + (NORM == 1 ? 0 : (h < H ? h : h - H) * a.dp) + d, w);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] *= f * w[j];
      } else if (h < H && temp != 1.f) {
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] *= temp;
      }
      if (cs != nullptr && !is_v) rotate_pairs(v, d, a.rot_dims, cs);
      if (h < H) st8(q + h * a.dp + d, v);
      else if (slot >= 0) st8(is_v ? vc + (h - H - G) * a.vp + d : kc + (h - H) * a.dp + d, v);
    }
  }
}

// Portions of prompts with a convolution and no norm over the whole projection: a group of S lanes takes one head (at most
// S * 8 channels) of PREP_ROWS consecutive rows. Where they and the rows before them belong to one sequence (nearly
// everywhere) all rows are requested at once and a window of them slides; elsewhere rows are convolved one by one.
constexpr int PREP_ROWS = 4;        // (eight rows, or three CTAs per SM, were 15 to 25 % slower)

template <typename T, bool NORM, int TAPS, int S>
__global__ void __launch_bounds__(256, 2)
qkv_prep_strip_kernel(const PrepArgs a) {
  __shared__ float temp_s[PREP_ROWS];
  const int H = a.heads, G = a.kv_heads, nq = H * a.dp, nk = G * a.dp, channels = nq + nk + G * a.vp;
  const int sub = threadIdx.x & (S - 1), h = blockIdx.y * (blockDim.x / S) + threadIdx.x / S;
  const bool there = h < H + 2 * G, is_v = h >= H + G;
  const int width = is_v ? a.vp : a.dp;
  const int base = is_v ? nq + nk + (h - H - G) * a.vp : h * a.dp;
  const int d = sub * 8;
  const bool mine = there && d < width;                  // (the other lanes take part in the sums with zeros)
  const int t0 = blockIdx.x * PREP_ROWS, n = min(PREP_ROWS, a.T - t0);
  const bool strip = t0 >= TAPS - 1 && n == PREP_ROWS && a.row_seq[t0 - (TAPS - 1)] == a.row_seq[t0 + PREP_ROWS - 1];
  const T* p = reinterpret_cast<const T*>(a.p) + base + d;
  Raw8<T> raw[TAPS - 1 + PREP_ROWS];
  float2 w[TAPS][4];
  if (strip && mine) {
#pragma unroll
    for (int i = 0; i < TAPS - 1 + PREP_ROWS; ++i) raw[i] = ld8raw<true>(p + (t0 - (TAPS - 1) + i) * a.ldp, 8);
#pragma unroll
    for (int k = 0; k < TAPS; ++k) {
      float v[8];
      ld8(reinterpret_cast<const T*>(a.conv_w) + static_cast<long long>(k) * channels + base + d, v);
#pragma unroll
      for (int j = 0; j < 4; ++j) w[k][j] = make_float2(v[2 * j], v[2 * j + 1]);
    }
  }
  if (threadIdx.x < n) temp_s[threadIdx.x] = a.temp_coef != 0.f ? query_temperature(a, t0 + threadIdx.x) : 1.f;
  const float inv_dim = 1.f / static_cast<float>(a.dim);
  float g[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) g[j] = 1.f;
  if (NORM && mine && !is_v) ld8(reinterpret_cast<const T*>(h < H ? a.wq : a.wk) + d, g);
  float2 win[TAPS][4];
  __syncthreads();
#pragma unroll
  for (int i = 0; i < TAPS - 1 + PREP_ROWS; ++i) {
    if (strip && mine) {
#pragma unroll
      for (int j = 0; j < 4; ++j) win[i % TAPS][j] = make_float2(ld1(&raw[i].v[2 * j]), ld1(&raw[i].v[2 * j + 1]));
    }
    const int r = i - (TAPS - 1);
    if (r < 0 || r >= n) continue;                       // the same for the whole CTA
    const int t = t0 + r;
    float v[8];
    if (!mine) {
#pragma unroll
      for (int j = 0; j < 8; ++j) v[j] = 0.f;
    } else if (strip) {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float2 y = make_float2(0.f, 0.f);
#pragma unroll
        for (int k = 0; k < TAPS; ++k) y = fma2(win[(r + k) % TAPS][j], w[k][j], y);
        v[2 * j] = y.x;
        v[2 * j + 1] = y.y;
      }
    } else {
      const int b = a.row_seq[t], start = a.cu_q[b];
      prep_load<T, true, false>(a, t, b, start, a.kv_lens[b] > a.cu_q[b + 1] - start, channels, base + d, v);
    }
    float f = 1.f;
    if (NORM) {
      float s = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) s += v[j] * v[j];
#pragma unroll
      for (int o = S / 2; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
      if (!is_v) f = rsqrtf(s * inv_dim + a.eps);
    }
    if (!mine) continue;
    if (h < H) f *= temp_s[r];
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] *= f * g[j];
    if (h < H) {
      st8(reinterpret_cast<T*>(a.q) + t * a.ldq + h * a.dp + d, v);
    } else {
      const long long slot = a.cache_slots[t];
      if (slot < 0) continue;
      if (is_v) st8(reinterpret_cast<T*>(a.v_cache) + (slot * G + (h - H - G)) * a.vp + d, v);
      else st8(reinterpret_cast<T*>(a.k_cache) + (slot * G + (h - H)) * a.dp + d, v);
    }
  }
}

template <typename T, bool NORM, int S>
static void launch_strip(const PrepArgs& a, int threads, dim3 grid, cudaStream_t stream) {
#define TW_CASE(K) case K: qkv_prep_strip_kernel<T, NORM, K, S><<<grid, threads, 0, stream>>>(a); break;
  switch (a.taps) { TW_CASE(1) TW_CASE(2) TW_CASE(3) TW_CASE(4) TW_CASE(5) TW_CASE(6) }
#undef TW_CASE
}

template <typename T, int S>
static void launch_prep(const PrepArgs& a, int norm, cudaStream_t stream) {
  const int heads = a.heads + 2 * a.kv_heads;
  int threads = (heads * S + 31) / 32 * 32;
  if (threads > 256) threads = 256;
  if (a.conv_w != nullptr && !a.single && norm != 2 && (norm == 0 || a.wq != nullptr) && a.cos_sin == nullptr && a.taps <= 6 && a.dp <= S * 8 && a.vp <= S * 8) {
    const dim3 grid((a.T + PREP_ROWS - 1) / PREP_ROWS, (heads * S + threads - 1) / threads);
    if (norm == 1) launch_strip<T, true, S>(a, threads, grid, stream);
    else launch_strip<T, false, S>(a, threads, grid, stream);
    return;
  }
#define TW_GO(N)                                                                             \
  do {                                                                                       \
    if (a.conv_w != nullptr) qkv_prep_kernel<T, N, true, S><<<a.T, threads, 0, stream>>>(a); \
    else qkv_prep_kernel<T, N, false, S><<<a.T, threads, 0, stream>>>(a);                    \
  } while (0)
  if (norm == 0) TW_GO(0);
  else if (norm == 1) TW_GO(1);
  else TW_GO(2);
#undef TW_GO
}

// ---- single query rows on SIMT -------------------------------------------------------------------------------------
constexpr int ROWS_THREADS = 128;      // and keys per round
constexpr int ROWS_VPT = 4;            // value columns per thread

struct RowsArgs {
  const void* q; long long ldq;
  const void *k_cache, *v_cache; int page;
  void* out; long long ldo;
  const int *tok_row, *tok_seq, *tok_kvlen, *block_table; int max_blocks;
  int heads, kv_heads, dp, vp;
  float scale;
  const float* slopes;
  int sink;
  float out_scale;
  int window, keep;          // window > 0: a query sees the last `window` keys (itself among them) and the first `keep`
  const float* key_bias;     // [heads]: weights sigmoid(scaled score + bias), not normalized; null: softmax
  int chunk;                 // > 0: a query sees the keys of its own chunk of that many positions
  const void* gate; long long ldg;      // [rows, heads]: the result times its sigmoid; null: off
};

template <typename T>
__global__ void __launch_bounds__(ROWS_THREADS)
attn_rows_kernel(const RowsArgs a) {
  extern __shared__ float rows_smem[];
  float* q_s = rows_smem;                              // [dp]
  __shared__ float p_s[ROWS_THREADS];
  __shared__ int slot_s[ROWS_THREADS];
  __shared__ float red[32];
  const int tok = blockIdx.x, h = blockIdx.y, g = h / (a.heads / a.kv_heads);
  const int row = a.tok_row[tok], kv_len = a.tok_kvlen[tok];
  const int* table = a.block_table + static_cast<long long>(a.tok_seq[tok]) * a.max_blocks;
  const T* q = reinterpret_cast<const T*>(a.q) + row * a.ldq + h * a.dp;
  for (int i = threadIdx.x; i < a.dp; i += ROWS_THREADS) q_s[i] = ld1(q + i);
  const float slope = a.slopes != nullptr ? a.slopes[h] : 0.f;
  const bool sigmoid = a.key_bias != nullptr;
  const float key_bias = sigmoid ? a.key_bias[h] : 0.f;
  const T* kc = reinterpret_cast<const T*>(a.k_cache);
  const T* vc = reinterpret_cast<const T*>(a.v_cache);
  float m = -INFINITY, l = 0.f, acc[ROWS_VPT];
#pragma unroll
  for (int c = 0; c < ROWS_VPT; ++c) acc[c] = 0.f;
  // the visible keys: `kept` first ones, then those from `from` on
  const int from = a.chunk > 0 ? (kv_len - 1) / a.chunk * a.chunk : a.window > 0 ? max(0, kv_len - a.window) : 0;
  const int kept = min(a.keep, from);
  const int visible = kept + kv_len - from;
  __syncthreads();
  for (int j0 = 0; j0 < visible; j0 += ROWS_THREADS) {
    const int i0 = j0 + threadIdx.x, n = min(ROWS_THREADS, visible - j0);
    float s = -INFINITY;
    if (i0 < visible) {
      const int j = i0 < kept ? i0 : i0 - kept + from;
      const int slot = table[j / a.page] * a.page + j % a.page;
      slot_s[threadIdx.x] = slot;
      const T* k = kc + (static_cast<long long>(slot) * a.kv_heads + g) * a.dp;
      float dot = 0.f;
      for (int d = 0; d < a.dp; d += 8) {
        float v[8];
        ld8(k + d, v);
#pragma unroll
        for (int e = 0; e < 8; ++e) dot = fmaf(q_s[d + e], v[e], dot);
      }
      s = dot * a.scale - slope * static_cast<float>(kv_len - 1 - j);
    }
    float p, alpha = 1.f;
    if (sigmoid) {
      p = i0 < visible ? sigmoid_f(s + key_bias) : 0.f;
    } else {
      float mx = warp_max(s);
      if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = mx;
      __syncthreads();
      mx = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
      const float m_new = fmaxf(m, mx);
      alpha = expf(m - m_new);        // 0 in the first round
      m = m_new;
      p = i0 < visible ? expf(s - m_new) : 0.f;
      l = l * alpha + p;
    }
    p_s[threadIdx.x] = p;
    __syncthreads();
#pragma unroll
    for (int c = 0; c < ROWS_VPT; ++c) {
      const int d = threadIdx.x + c * ROWS_THREADS;
      if (d >= a.vp) continue;
      float x = acc[c] * alpha;
      for (int i = 0; i < n; ++i)
        x = fmaf(p_s[i], ld1(vc + (static_cast<long long>(slot_s[i]) * a.kv_heads + g) * a.vp + d), x);
      acc[c] = x;
    }
    __syncthreads();
  }
  float inv = a.out_scale;
  if (!sigmoid) {
    float tot[1] = {l};
    block_sum<1>(tot, red);
    if (a.sink) tot[0] += expf(-m);
    inv /= tot[0];
  }
  if (a.gate != nullptr) inv *= sigmoid_f(ld1(reinterpret_cast<const T*>(a.gate) + row * a.ldg + h));
  T* o = reinterpret_cast<T*>(a.out) + row * a.ldo + h * a.vp;
#pragma unroll
  for (int c = 0; c < ROWS_VPT; ++c) {
    const int d = threadIdx.x + c * ROWS_THREADS;
    if (d < a.vp) st1(o + d, acc[c] * inv);
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

extern "C" int tw_qkv_prep(const void* p, long long ldp, int T, int heads, int kv_heads, int dim, int dp, int vp, void* q,
                           long long ldq, void* k_cache, void* v_cache, const int* positions, const int* cache_slots,
                           const void* conv_w, void* conv_state, int taps, const int* row_seq, const int* cu_q,
                           const int* kv_lens, const int* slots, int n_seqs, int single, int norm, const void* wq,
                           const void* wk, float eps, float temp_coef, int temp_every, const float* cos_sin, int rot_dims,
                           int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (dp % 8 != 0 || vp % 8 != 0 || ldp % 8 != 0 || ldq % 8 != 0 || !aligned16(p) || !aligned16(q) || !aligned16(k_cache) ||
      !aligned16(v_cache) || !aligned16(conv_w) || !aligned16(conv_state) || !aligned16(wq) || !aligned16(wk)) {
    set_last_error("qkv_prep: heads of %d and %d elements in rows of %lld: multiples of eight on 16-byte boundaries are needed",
                   dp, vp, ldp);
    return 1;
  }
  if (cos_sin != nullptr && (rot_dims % 2 != 0 || rot_dims <= 0 || rot_dims > dim || !aligned16(cos_sin))) {
    set_last_error("qkv_prep: %d rotated dimensions of %d", rot_dims, dim);
    return 1;
  }
  if (heads <= 0 || kv_heads < 0 || (kv_heads > 0 && (k_cache == nullptr || v_cache == nullptr)) || norm < 0 || norm > 2 ||
      (wq == nullptr) != (wk == nullptr) || (norm == 2 && wq == nullptr) ||
      temp_every <= 0 || (conv_w != nullptr && (row_seq == nullptr || taps < 1)) ||
      (conv_w != nullptr && taps > 1 && (conv_state == nullptr || slots == nullptr))) {
    set_last_error("qkv_prep: bad arguments (heads=%d, kv_heads=%d, norm=%d, taps=%d)", heads, kv_heads, norm, taps);
    return 1;
  }
  const PrepArgs a{p, ldp, T, heads, kv_heads, dim, dp, vp, q, ldq, k_cache, v_cache, positions, cache_slots, conv_w,
                   conv_state, taps, row_seq, cu_q, kv_lens, slots, single, wq, wk, eps, temp_coef, temp_every, cos_sin, rot_dims};
  const int wide = dp > vp ? dp : vp;
#define TW_GO(T)                                          \
  do {                                                    \
    if (wide <= 32) launch_prep<T, 4>(a, norm, stream);   \
    else if (wide <= 64) launch_prep<T, 8>(a, norm, stream);   \
    else if (wide <= 128) launch_prep<T, 16>(a, norm, stream); \
    else launch_prep<T, 32>(a, norm, stream);             \
  } while (0)
  if (dtype == TW_BF16) TW_GO(__nv_bfloat16);
  else TW_GO(float);
#undef TW_GO
  if (check_launch("qkv_prep")) return 1;
  if (conv_w != nullptr && taps > 1 && !single)
    return tw_conv_state(p, ldp, conv_state, cu_q, kv_lens, slots, n_seqs, heads * dp + kv_heads * (dp + vp), taps, dtype,
                         stream);
  return 0;
}

extern "C" int tw_attn_rows(const void* q, long long ldq, const void* k_cache, const void* v_cache, int page, void* out,
                            long long ldo, const int* tok_row, const int* tok_seq, const int* tok_kvlen, int n,
                            const int* block_table, int max_blocks, int heads, int kv_heads, int dp, int vp, float scale,
                            const float* slopes, int sink, float out_scale, int window, int keep, const float* key_bias,
                            int chunk, const void* gate, long long ldg, int dtype, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (dp % 8 != 0 || dp > 4096 || vp > ROWS_VPT * ROWS_THREADS || kv_heads <= 0 || heads % kv_heads != 0 ||
      !aligned16(k_cache)) {
    set_last_error("attn_rows: unsupported shape (queries and keys of %d, values of %d elements, %d / %d heads)", dp, vp, heads,
                   kv_heads);
    return 1;
  }
  const RowsArgs a{q, ldq, k_cache, v_cache, page, out, ldo, tok_row, tok_seq, tok_kvlen, block_table, max_blocks, heads,
                   kv_heads, dp, vp, scale, slopes, sink, out_scale, window, keep, key_bias, chunk, gate, ldg};
  const dim3 grid(n, heads);
  if (dtype == TW_BF16) attn_rows_kernel<__nv_bfloat16><<<grid, ROWS_THREADS, dp * 4, stream>>>(a);
  else attn_rows_kernel<float><<<grid, ROWS_THREADS, dp * 4, stream>>>(a);
  return check_launch("attn_rows");
}
