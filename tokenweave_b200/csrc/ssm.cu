// State-space (Mamba-2) kernels for bf16 and fp32 activations and any sizes; the recurrent state is always fp32.
//
// A step's rows are sequences laid out back to back (cu_q); sequence b continues the state in slot slots[b] when it
// has tokens behind it (kv_lens[b] > its rows in this step) and starts from zeros otherwise, whatever the slot holds.
//
//   tw_causal_conv       per-channel causal convolution with bias and silu. The taps - 1 inputs before a sequence's
//                        first row come from its convolution state [slot, taps - 1, channels] (oldest first), which
//                        is moved on by the second launch; a step of single-token sequences does both in one launch
//   tw_conv_state        the second launch alone, for kernels that convolve on their own
//   tw_ssd_scan          token-by-token recurrence S <- exp(-exp(A) dt) S + dt B x^T, y = S^T C + D x, dt =
//                        softplus(raw + bias): decoding, short portions, fp32
//   tw_decay_scan        the same with unit steps, a given decay per head and no skip (lightning attention: x = values,
//                        B = keys, C = queries, every head a group of its own)
//
// State layout [slot, head, vdim, state]: a warp owns rows of vdim, its lanes the state dimension.
#include "tw_host.h"
#include "tw_kernels.h"
#include "tw_typed.cuh"

namespace tw {

constexpr int CONV_MAX_TAPS = 8;
constexpr int CONV_ROWS = 8;       // rows per thread

struct ConvArgs {
  const void* x; long long ldx;       // inputs [T, channels]
  const void* w;                      // [taps, channels]: tap-major, last tap = current token
  const void* bias;
  void* state;                        // [slots, taps - 1, channels]
  void* out; long long ldo;
  const int* row_seq; const int* cu_q; const int* kv_lens; const int* slots;
  int T, n_seqs, channels, taps;
};

__device__ __forceinline__ bool has_past(const ConvArgs& a, int b) {
  return a.kv_lens[b] > a.cu_q[b + 1] - a.cu_q[b];
}

// the input `back` tokens before row t of sequence b (back may reach before the rows of this step)
template <typename T, bool VEC>
__device__ __forceinline__ void conv_input(const ConvArgs& a, int b, int t, int back, int c, float (&v)[8]) {
  const int start = a.cu_q[b];
  const int r = t - back;
  if (r >= start) {
    ld8n<VEC>(reinterpret_cast<const T*>(a.x) + r * a.ldx + c, a.channels - c, v);
  } else if (has_past(a, b)) {
    const int k = a.taps - 1 - (start - r);
    ld8n<VEC>(reinterpret_cast<const T*>(a.state) +
                  (static_cast<long long>(a.slots[b]) * (a.taps - 1) + k) * a.channels + c,
              a.channels - c, v);
  } else {
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = 0.f;
  }
}

// A thread owns eight channels of CONV_ROWS consecutive rows. Where they and the rows before them belong to one sequence
// (nearly everywhere) all rows are requested at once and a window of converted inputs slides over them; the rest takes
// the general path row by row.
template <typename T, bool VEC, int TAPS>
__global__ void __launch_bounds__(128)
causal_conv_kernel(const ConvArgs a) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (c >= a.channels) return;
  const int n_ch = a.channels - c;
  const int t0 = blockIdx.y * CONV_ROWS;
  const T* xp = reinterpret_cast<const T*>(a.x) + c;
  T* op = reinterpret_cast<T*>(a.out) + c;
  const T* wp = reinterpret_cast<const T*>(a.w) + c;
  if (t0 >= TAPS - 1 && t0 + CONV_ROWS <= a.T && a.row_seq[t0 - (TAPS - 1)] == a.row_seq[t0 + CONV_ROWS - 1]) {
    Raw8<T> raw[TAPS - 1 + CONV_ROWS];
#pragma unroll
    for (int i = 0; i < TAPS - 1 + CONV_ROWS; ++i) raw[i] = ld8raw<VEC>(xp + (t0 - (TAPS - 1) + i) * a.ldx, n_ch);
    float2 w[TAPS][4], bias[4], win[TAPS][4];        // win[i % TAPS]: input of row i of the strip
    float v[8];
#pragma unroll
    for (int k = 0; k < TAPS; ++k) {
      ld8n<VEC>(wp + static_cast<long long>(k) * a.channels, n_ch, v);
#pragma unroll
      for (int j = 0; j < 4; ++j) w[k][j] = make_float2(v[2 * j], v[2 * j + 1]);
    }
    ld8n<VEC>(reinterpret_cast<const T*>(a.bias) + c, n_ch, v);
#pragma unroll
    for (int j = 0; j < 4; ++j) bias[j] = make_float2(v[2 * j], v[2 * j + 1]);
#pragma unroll
    for (int i = 0; i < TAPS - 1 + CONV_ROWS; ++i) {
#pragma unroll
      for (int j = 0; j < 4; ++j) win[i % TAPS][j] = make_float2(ld1(&raw[i].v[2 * j]), ld1(&raw[i].v[2 * j + 1]));
      if (i < TAPS - 1) continue;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float2 y = bias[j];
#pragma unroll
        for (int k = 0; k < TAPS; ++k) y = fma2(win[(i - (TAPS - 1) + k) % TAPS][j], w[k][j], y);
        v[2 * j] = silu_t<T>(y.x);
        v[2 * j + 1] = silu_t<T>(y.y);
      }
      st8n<VEC>(op + (t0 + i - (TAPS - 1)) * a.ldo, n_ch, v);
    }
    return;
  }
  const int t_end = min(a.T, t0 + CONV_ROWS);
#pragma unroll 1
  for (int t = t0; t < t_end; ++t) {
    float y[8];
    ld8n<VEC>(reinterpret_cast<const T*>(a.bias) + c, n_ch, y);
#pragma unroll 1
    for (int k = 0; k < TAPS; ++k) {
      float v[8], w[8];
      conv_input<T, VEC>(a, a.row_seq[t], t, TAPS - 1 - k, c, v);
      ld8n<VEC>(wp + static_cast<long long>(k) * a.channels, n_ch, w);
#pragma unroll
      for (int j = 0; j < 8; ++j) y[j] = fmaf(v[j], w[j], y[j]);
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) y[j] = silu_t<T>(y[j]);
    st8n<VEC>(op + t * a.ldo, n_ch, y);
  }
}

// Moves every sequence's convolution state on: the new state's entry k is the input taps - 1 - k tokens before the
// next token. Entries are written oldest first and only read further along, so one thread works in place.
template <typename T, bool VEC>
__global__ void __launch_bounds__(128)
conv_state_kernel(const ConvArgs a) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (c >= a.channels) return;
  const int b = blockIdx.y;
  const int end = a.cu_q[b + 1];
  T* st = reinterpret_cast<T*>(a.state) + static_cast<long long>(a.slots[b]) * (a.taps - 1) * a.channels + c;
  for (int k = 0; k < a.taps - 1; ++k) {
    float v[8];
    conv_input<T, VEC>(a, b, end, a.taps - 1 - k, c, v);
    st8n<VEC>(st + static_cast<long long>(k) * a.channels, a.channels - c, v);
  }
}

// One token per sequence: convolution and state in one launch.
template <typename T, bool VEC, int TAPS>
__global__ void __launch_bounds__(128)
causal_conv_step_kernel(const ConvArgs a) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (c >= a.channels) return;
  const int b = blockIdx.y, t = a.cu_q[b];
  float h[TAPS][8], y[8];
#pragma unroll
  for (int k = 0; k < TAPS; ++k) conv_input<T, VEC>(a, b, t, TAPS - 1 - k, c, h[k]);     // oldest first
  ld8n<VEC>(reinterpret_cast<const T*>(a.bias) + c, a.channels - c, y);
#pragma unroll
  for (int k = 0; k < TAPS; ++k) {
    float w[8];
    ld8n<VEC>(reinterpret_cast<const T*>(a.w) + static_cast<long long>(k) * a.channels + c, a.channels - c, w);
#pragma unroll
    for (int j = 0; j < 8; ++j) y[j] = fmaf(h[k][j], w[j], y[j]);
  }
#pragma unroll
  for (int j = 0; j < 8; ++j) y[j] = silu_t<T>(y[j]);
  st8n<VEC>(reinterpret_cast<T*>(a.out) + t * a.ldo + c, a.channels - c, y);
  T* st = reinterpret_cast<T*>(a.state) + static_cast<long long>(a.slots[b]) * (TAPS - 1) * a.channels + c;
#pragma unroll
  for (int k = 0; k + 1 < TAPS; ++k) st8n<VEC>(st + static_cast<long long>(k) * a.channels, a.channels - c, h[k + 1]);
}

// ---- recurrence, token by token --------------------------------------------------------------------------
struct ScanArgs {
  const void* xbc; long long ldx;              // [T, heads * vdim | groups * state | groups * state]
  const void* dt; long long ldt;               // [T, heads] raw step sizes
  const void* dt_bias; const void* A_log; const void* D;    // [heads]; unused with `decay`
  const float* decay;                          // [heads]: fixed decays, unit steps and no skip (dt may be null)
  float* state;                                // [slots, heads, vdim, state]
  void* y; long long ldy;                      // [T, heads * vdim]
  const int* seqs;                             // sequences of this launch
  const int* cu_q; const int* kv_lens; const int* slots;
  int heads, vdim, N, groups;
};

constexpr int SCAN_WARPS = 4;

template <typename T, int NK, int PW>
__global__ void __launch_bounds__(SCAN_WARPS * 32)
ssd_scan_kernel(const ScanArgs a) {
  const int b = a.seqs[blockIdx.x], h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int p0 = (blockIdx.z * SCAN_WARPS + warp) * PW;
  if (p0 >= a.vdim) return;
  const int t0 = a.cu_q[b], t1 = a.cu_q[b + 1];
  const bool past = a.kv_lens[b] > t1 - t0;
  float* st = a.state + ((static_cast<long long>(a.slots[b]) * a.heads + h) * a.vdim + p0) * a.N;
  float S[PW][NK];
#pragma unroll
  for (int p = 0; p < PW; ++p)
#pragma unroll
    for (int k = 0; k < NK; ++k) {
      const int n = lane + 32 * k;
      S[p][k] = (past && p0 + p < a.vdim && n < a.N) ? st[static_cast<long long>(p) * a.N + n] : 0.f;
    }
  const bool fixed = a.decay != nullptr;
  const float bias = fixed ? 0.f : ld1(reinterpret_cast<const T*>(a.dt_bias) + h);
  const float A = fixed ? 0.f : expf(ld1(reinterpret_cast<const T*>(a.A_log) + h));
  const float D = fixed ? 0.f : ld1(reinterpret_cast<const T*>(a.D) + h);
  const int g = h / (a.heads / a.groups);
  const int off_b = a.heads * a.vdim + g * a.N, off_c = off_b + a.groups * a.N;
  for (int t = t0; t < t1; ++t) {
    const T* xr = reinterpret_cast<const T*>(a.xbc) + t * a.ldx;
    float B[NK], C[NK], x[PW], y[PW];
#pragma unroll
    for (int k = 0; k < NK; ++k) {
      const int n = lane + 32 * k;
      B[k] = n < a.N ? ld1(xr + off_b + n) : 0.f;
      C[k] = n < a.N ? ld1(xr + off_c + n) : 0.f;
    }
#pragma unroll
    for (int p = 0; p < PW; ++p) x[p] = p0 + p < a.vdim ? ld1(xr + h * a.vdim + p0 + p) : 0.f;
    const float dt = fixed ? 1.f : softplus_f(ld1(reinterpret_cast<const T*>(a.dt) + t * a.ldt + h) + bias);
    const float decay = fixed ? a.decay[h] : expf(-A * dt);
#pragma unroll
    for (int p = 0; p < PW; ++p) {
      const float dx = dt * x[p];
      y[p] = 0.f;
#pragma unroll
      for (int k = 0; k < NK; ++k) {
        S[p][k] = fmaf(decay, S[p][k], dx * B[k]);
        y[p] = fmaf(S[p][k], C[k], y[p]);
      }
    }
#pragma unroll
    for (int p = 0; p < PW; ++p) y[p] = warp_sum(y[p]);
    if (lane == 0) {
      T* yr = reinterpret_cast<T*>(a.y) + t * a.ldy + h * a.vdim + p0;
#pragma unroll
      for (int p = 0; p < PW; ++p)
        if (p0 + p < a.vdim) st1(yr + p, fmaf(D, x[p], y[p]));
    }
  }
#pragma unroll
  for (int p = 0; p < PW; ++p)
#pragma unroll
    for (int k = 0; k < NK; ++k) {
      const int n = lane + 32 * k;
      if (p0 + p < a.vdim && n < a.N) st[static_cast<long long>(p) * a.N + n] = S[p][k];
    }
}

static int check_launch(const char* what) {
  const cudaError_t e = cudaGetLastError();
  if (e == cudaSuccess) return 0;
  set_last_error("%s launch failed: %s", what, cudaGetErrorString(e));
  return 1;
}
static bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename T, bool VEC>
static int launch_conv(const ConvArgs& a, int single, cudaStream_t stream) {
  const int groups = (a.channels + 7) / 8;
  const int threads = groups >= 128 ? 128 : (groups + 31) / 32 * 32;
  const int gx = (groups + threads - 1) / threads;
  if (single) {
    const dim3 grid(gx, a.n_seqs);
#define TW_CASE(K) case K: causal_conv_step_kernel<T, VEC, K><<<grid, threads, 0, stream>>>(a); break;
    switch (a.taps) { TW_CASE(1) TW_CASE(2) TW_CASE(3) TW_CASE(4) TW_CASE(5) TW_CASE(6) TW_CASE(7) TW_CASE(8) }
#undef TW_CASE
    return check_launch("causal_conv (single tokens)");
  }
  const dim3 grid(gx, (a.T + CONV_ROWS - 1) / CONV_ROWS);
#define TW_CASE(K) case K: causal_conv_kernel<T, VEC, K><<<grid, threads, 0, stream>>>(a); break;
  switch (a.taps) { TW_CASE(1) TW_CASE(2) TW_CASE(3) TW_CASE(4) TW_CASE(5) TW_CASE(6) TW_CASE(7) TW_CASE(8) }
#undef TW_CASE
  if (check_launch("causal_conv")) return 1;
  if (a.taps > 1) {
    conv_state_kernel<T, VEC><<<dim3(gx, a.n_seqs), threads, 0, stream>>>(a);
    return check_launch("causal_conv (state)");
  }
  return 0;
}

template <typename T>
static int launch_scan(const ScanArgs& a, int n_seqs, cudaStream_t stream) {
#define TW_GO(NK, PW)                                                                            \
  do {                                                                                           \
    const dim3 grid(n_seqs, a.heads, (a.vdim + SCAN_WARPS * PW - 1) / (SCAN_WARPS * PW));        \
    ssd_scan_kernel<T, NK, PW><<<grid, SCAN_WARPS * 32, 0, stream>>>(a);                         \
  } while (0)
  if (a.N <= 32) TW_GO(1, 4);
  else if (a.N <= 64) TW_GO(2, 4);
  else if (a.N <= 128) TW_GO(4, 4);
  else if (a.N <= 256) TW_GO(8, 4);
  else if (a.N <= 512) TW_GO(16, 2);
  else {
    set_last_error("ssd_scan: states of up to 512 dimensions are supported (got %d)", a.N);
    return 1;
  }
#undef TW_GO
  return check_launch("ssd_scan");
}

}  // namespace tw

using namespace tw;

extern "C" int tw_causal_conv(const void* x, long long ldx, const void* w, const void* bias, void* state, void* out,
                              long long ldo, const int* row_seq, const int* cu_q, const int* kv_lens, const int* slots,
                              int T, int n_seqs, int channels, int taps, int single, int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (taps < 1 || taps > CONV_MAX_TAPS) {
    set_last_error("causal_conv: 1 to %d taps are supported (got %d)", CONV_MAX_TAPS, taps);
    return 1;
  }
  const ConvArgs a{x, ldx, w, bias, state, out, ldo, row_seq, cu_q, kv_lens, slots, T, n_seqs, channels, taps};
  const bool vec = ldx % 8 == 0 && ldo % 8 == 0 && channels % 8 == 0 && aligned16(x) && aligned16(w) && aligned16(bias) &&
                   aligned16(state) && aligned16(out);
  if (dtype == TW_BF16)
    return vec ? launch_conv<__nv_bfloat16, true>(a, single, stream) : launch_conv<__nv_bfloat16, false>(a, single, stream);
  return vec ? launch_conv<float, true>(a, single, stream) : launch_conv<float, false>(a, single, stream);
}

extern "C" int tw_ssd_scan(const void* xbc, long long ldx, const void* dt, long long ldt, const void* dt_bias,
                           const void* A_log, const void* D, float* state, void* y, long long ldy, const int* seqs,
                           int n_seqs, const int* cu_q, const int* kv_lens, const int* slots, int heads, int vdim, int N,
                           int groups, int dtype, cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  if (groups <= 0 || heads % groups != 0) {
    set_last_error("ssd_scan: %d heads do not divide into %d groups", heads, groups);
    return 1;
  }
  const ScanArgs a{xbc, ldx, dt, ldt, dt_bias, A_log, D, nullptr, state, y, ldy, seqs, cu_q, kv_lens, slots, heads, vdim, N, groups};
  return dtype == TW_BF16 ? launch_scan<__nv_bfloat16>(a, n_seqs, stream) : launch_scan<float>(a, n_seqs, stream);
}

extern "C" int tw_decay_scan(const void* vkq, long long ldx, const float* decay, float* state, void* y, long long ldy,
                             const int* seqs, int n_seqs, const int* cu_q, const int* kv_lens, const int* slots, int heads,
                             int vdim, int N, int dtype, cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  const ScanArgs a{vkq, ldx, nullptr, 0, nullptr, nullptr, nullptr, decay, state, y, ldy, seqs, cu_q, kv_lens, slots,
                   heads, vdim, N, heads};
  return dtype == TW_BF16 ? launch_scan<__nv_bfloat16>(a, n_seqs, stream) : launch_scan<float>(a, n_seqs, stream);
}

extern "C" int tw_conv_state(const void* x, long long ldx, void* state, const int* cu_q, const int* kv_lens,
                             const int* slots, int n_seqs, int channels, int taps, int dtype, cudaStream_t stream) {
  if (n_seqs <= 0 || taps <= 1) return 0;
  const ConvArgs a{x, ldx, nullptr, nullptr, state, nullptr, 0, nullptr, cu_q, kv_lens, slots, 0, n_seqs, channels, taps};
  const bool vec = ldx % 8 == 0 && channels % 8 == 0 && aligned16(x) && aligned16(state);
  const int groups = (channels + 7) / 8;
  const int threads = groups >= 128 ? 128 : (groups + 31) / 32 * 32;
  const dim3 grid((groups + threads - 1) / threads, n_seqs);
  if (dtype == TW_BF16) {
    if (vec) conv_state_kernel<__nv_bfloat16, true><<<grid, threads, 0, stream>>>(a);
    else conv_state_kernel<__nv_bfloat16, false><<<grid, threads, 0, stream>>>(a);
  } else {
    if (vec) conv_state_kernel<float, true><<<grid, threads, 0, stream>>>(a);
    else conv_state_kernel<float, false><<<grid, threads, 0, stream>>>(a);
  }
  return check_launch("conv_state");
}
