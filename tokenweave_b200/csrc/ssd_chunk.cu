// State-space (Mamba-2) recurrence of long runs of tokens on the tensor cores: 64 tokens at a time in the quadratic
// form, the state carried from chunk to chunk.
//
// With l_i the running sum of log-decays inside a chunk, per head:
//     y_i   = sum_{j <= i} (C_i . B_j) exp(l_i - l_j) dt_j x_j  +  exp(l_i) C_i S  +  D x_i
//     S     = exp(l_last) S + sum_j exp(l_last - l_j) dt_j x_j B_j^T
// B, C, x are bf16 activations and enter the products exactly. Everything of the recurrence is fp32: the running sums
// are formed in double and kept as two floats (differences of nearby sums stay accurate behind strong decays), and
// the three fp32 operands of products - the state, the weighted scores, the weighted inputs - are split into two
// bf16 terms each.
//
// One CTA (16 warps) per sequence, head and 64 rows of vdim. The state lives in accumulator registers for the whole
// sequence and passes through shared memory once per chunk as the operand of C S; the next chunk's B, C and x arrive by
// cp.async meanwhile. A chunk has two phases between barriers: the weighted scores (ten warps own one 16 x 16 tile of
// the lower triangle each), the weighted inputs and C S; then scores times x, the outputs, and the state. An earlier
// form with eight warps, in which every warp made the weights of its own rows in registers, took 2.3 times the
// instructions per scheduler slot (the weights were made twice) and was bound by latency.
#include "tw_host.h"
#include "tw_kernels.h"
#include "tw_mma.cuh"
#include "tw_typed.cuh"

namespace tw {

struct ChunkArgs {
  const __nv_bfloat16* xbc; long long ldx;       // [T, heads * vdim | groups * N | groups * N]
  const __nv_bfloat16* dt; long long ldt;        // [T, heads]
  const __nv_bfloat16 *dt_bias, *A_log, *D;      // [heads]; unused with `decay`
  const float* decay;                            // [heads]: fixed decays, unit steps, no skip
  float* state;                                  // [slots, heads, vdim, N]
  __nv_bfloat16* y; long long ldy;
  const int *seqs, *cu_q, *kv_lens, *slots;
  int heads, vdim, N, groups;
};

constexpr int CH_L = 64;          // tokens per chunk
constexpr int CH_P = 64;          // rows of vdim per CTA
constexpr int CH_THREADS = 512;

template <int NP>
struct ChunkSmem {
  static constexpr int BUFS = NP <= 128 ? 2 : 1;
  static constexpr int LDN = NP + 8, LDP = CH_P + 8;           // padded rows: conflict-free ldmatrix
  static constexpr int BC = CH_L * LDN, X = CH_L * LDP;        // elements
  static constexpr int STAGE = 2 * BC + X;
  static constexpr int S_ELEMS = CH_P * LDN;
  static constexpr int W_ELEMS = CH_L * LDP;                                 // weighted scores, weighted inputs
  static constexpr int BYTES = (BUFS * STAGE + 2 * S_ELEMS + 4 * W_ELEMS) * 2 + 2 * 4 * CH_L * 4;
};

// Running sums of one chunk by one warp: token 2 lane and 2 lane + 1 per lane.
struct ChunkSums {
  float dt[CH_L];      // step sizes, zero behind the run's end
  float hi[CH_L], lo[CH_L];
  float last[CH_L];    // exp(l_last - l_j) dt_j
};

// The raw step sizes of a chunk: requested a chunk ahead of chunk_sums (a row of the projection per token: nothing of it
// is in a cache).
__device__ __forceinline__ float2 chunk_steps(const ChunkArgs& a, int t0, int t_end, int h, int lane) {
  float2 r = make_float2(0.f, 0.f);
  const int t = t0 + 2 * lane;
  if (a.decay != nullptr) return r;
  if (t < t_end) r.x = ld1(a.dt + t * a.ldt + h);
  if (t + 1 < t_end) r.y = ld1(a.dt + (t + 1) * a.ldt + h);
  return r;
}

__device__ __forceinline__ void chunk_sums(ChunkSums* s, float2 raw, int n, float bias, double A, bool fixed, int lane) {
  double l[2];
  float d[2];
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    d[e] = 2 * lane + e >= n ? 0.f : fixed ? 1.f : softplus_f((e ? raw.y : raw.x) + bias);
    l[e] = -A * d[e];
  }
  double run = l[0] + l[1];
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const double up = __shfl_up_sync(0xffffffffu, run, o);
    if (lane >= o) run += up;
  }
  const double total = __shfl_sync(0xffffffffu, run, 31);
  const double v[2] = {run - l[1], run};
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int j = 2 * lane + e;
    const float hi = static_cast<float>(v[e]);
    s->dt[j] = d[e];
    s->hi[j] = hi;
    s->lo[j] = static_cast<float>(v[e] - static_cast<double>(hi));
    s->last[j] = expf(static_cast<float>(total - v[e])) * d[e];
  }
}

template <int NP>
__device__ __forceinline__ void chunk_load(const ChunkArgs& a, __nv_bfloat16* st, int t0, int n, int off_x, int p_valid,
                                           int off_b, int off_c) {
  using SM = ChunkSmem<NP>;
  __nv_bfloat16 *sb = st, *sc = st + SM::BC, *sx = st + 2 * SM::BC;
  for (int i = threadIdx.x; i < CH_L * (NP / 8); i += CH_THREADS) {
    const int r = i / (NP / 8), c = (i - r * (NP / 8)) * 8;
    const bool ok = r < n && c < a.N;
    const __nv_bfloat16* src = a.xbc + (t0 + (ok ? r : 0)) * a.ldx;
    cp_async16(sb + r * SM::LDN + c, src + off_b + (ok ? c : 0), ok ? 16 : 0);
    cp_async16(sc + r * SM::LDN + c, src + off_c + (ok ? c : 0), ok ? 16 : 0);
  }
  for (int i = threadIdx.x; i < CH_L * (CH_P / 8); i += CH_THREADS) {
    const int r = i >> 3, c = (i & 7) * 8;
    const bool ok = r < n && c < p_valid;
    cp_async16(sx + r * SM::LDP + c, a.xbc + (t0 + (ok ? r : 0)) * a.ldx + off_x + (ok ? c : 0), ok ? 16 : 0);
  }
  cp_async_commit();
}

template <int NP>
__global__ void __launch_bounds__(CH_THREADS, 1)
ssd_chunk_kernel(const ChunkArgs a) {
  using SM = ChunkSmem<NP>;
  constexpr int NT = NP / 32;                // 8-column tiles of this warp's quarter of the state dimension
  extern __shared__ __align__(16) uint8_t smem_raw[];
  __nv_bfloat16* stage = reinterpret_cast<__nv_bfloat16*>(smem_raw);
  __nv_bfloat16* s_hi = stage + SM::BUFS * SM::STAGE;        // state [vdim][N]
  __nv_bfloat16* s_lo = s_hi + SM::S_ELEMS;
  __nv_bfloat16* m_hi = s_lo + SM::S_ELEMS;                  // weighted scores [token][token]
  __nv_bfloat16* m_lo = m_hi + SM::W_ELEMS;
  __nv_bfloat16* w_hi = m_lo + SM::W_ELEMS;                  // weighted inputs [token][vdim]
  __nv_bfloat16* w_lo = w_hi + SM::W_ELEMS;
  ChunkSums* sums = reinterpret_cast<ChunkSums*>(w_lo + SM::W_ELEMS);     // [2]

  const int b = a.seqs[blockIdx.x], h = blockIdx.y, p0 = blockIdx.z * CH_P;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int wr = warp & 3, wq = warp >> 2;   // row group (tokens for y, vdim for the state) and quarter of the columns
  const int q4 = lane >> 2, q2 = (lane & 3) * 2;
  const int t_begin = a.cu_q[b], t_end = a.cu_q[b + 1];
  const int p_valid = min(CH_P, a.vdim - p0);
  const int g = h / (a.heads / a.groups);
  const int off_x = h * a.vdim + p0, off_b = a.heads * a.vdim + g * a.N, off_c = off_b + a.groups * a.N;
  const bool fixed = a.decay != nullptr;
  const float bias = fixed ? 0.f : ld1(a.dt_bias + h), D = fixed ? 0.f : ld1(a.D + h);
  const double A = fixed ? decay_rate(a.decay[h]) : static_cast<double>(expf(ld1(a.A_log + h)));
  // tile of the lower triangle this warp makes (warps 0..9)
  const int ti = warp < 1 ? 0 : warp < 3 ? 1 : warp < 6 ? 2 : 3, tj = warp - ti * (ti + 1) / 2;

  // state rows p = 16 wr + q4 (+ 8), columns n = wq NP/4 + 8 k + q2 (+ 1)
  float S[NT][4];
  float* st = a.state + ((static_cast<long long>(a.slots[b]) * a.heads + h) * a.vdim + p0) * a.N;
  const bool past = a.kv_lens[b] > t_end - t_begin;
#pragma unroll
  for (int k = 0; k < NT; ++k)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int p = 16 * wr + q4 + (e >> 1) * 8, n = wq * (NP / 4) + 8 * k + q2 + (e & 1);
      S[k][e] = (past && p < p_valid && n < a.N) ? st[static_cast<long long>(p) * a.N + n] : 0.f;
    }

  chunk_load<NP>(a, stage, t_begin, min(CH_L, t_end - t_begin), off_x, p_valid, off_b, off_c);
  float2 steps = make_float2(0.f, 0.f);      // warp 15: raw step sizes of the next chunk
  if (warp == 15) {
    steps = chunk_steps(a, t_begin, t_end, h, lane);
    chunk_sums(&sums[0], steps, t_end - t_begin, bias, A, fixed, lane);
    steps = chunk_steps(a, t_begin + CH_L, t_end, h, lane);
  }

  int c = 0;
  for (int t0 = t_begin; t0 < t_end; t0 += CH_L, ++c) {
    const int n_tok = min(CH_L, t_end - t0);
    __nv_bfloat16* cur = stage + (SM::BUFS == 2 ? (c & 1) : 0) * SM::STAGE;
    const __nv_bfloat16 *sb = cur, *sc = cur + SM::BC, *sx = cur + 2 * SM::BC;
    const ChunkSums& sm = sums[c & 1];
    // the state as the operand of C S
#pragma unroll
    for (int k = 0; k < NT; ++k) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        uint32_t hi, lo;
        split_bf16x2(S[k][2 * e], S[k][2 * e + 1], hi, lo);
        const int o = (16 * wr + q4 + 8 * e) * SM::LDN + wq * (NP / 4) + 8 * k + q2;
        *reinterpret_cast<uint32_t*>(s_hi + o) = hi;
        *reinterpret_cast<uint32_t*>(s_lo + o) = lo;
      }
    }
    cp_async_wait<0>();
    __syncthreads();
    const bool more = t0 + CH_L < t_end;
    if (SM::BUFS == 2 && more)
      chunk_load<NP>(a, stage + ((c + 1) & 1) * SM::STAGE, t0 + CH_L, min(CH_L, t_end - t0 - CH_L), off_x, p_valid, off_b,
                     off_c);

    // ---- phase 1: one tile of weighted scores per warp ----
    if (warp < 10) {
      float G[2][4] = {};
#pragma unroll
      for (int k = 0; k < NP; k += 16) {
        uint32_t fc[4], fb[4];
        ldmatrix_x4(fc, smem_u32(sc + 16 * ti * SM::LDN + k + frag_a(lane, SM::LDN)));
        ldmatrix_x4(fb, smem_u32(sb + 16 * tj * SM::LDN + k + frag_b(lane, SM::LDN)));
        mma_bf16(G[0], fc, fb[0], fb[1]);
        mma_bf16(G[1], fc, fb[2], fb[3]);
      }
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int i = 16 * ti + q4 + 8 * e;
        const float hi_i = sm.hi[i], lo_i = sm.lo[i];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int j = 16 * tj + 8 * half + q2;
          const float2 hj = *reinterpret_cast<const float2*>(sm.hi + j), lj = *reinterpret_cast<const float2*>(sm.lo + j);
          const float2 d = *reinterpret_cast<const float2*>(sm.dt + j);
          const float w0 = j <= i ? G[half][2 * e] * expf((hi_i - hj.x) + (lo_i - lj.x)) * d.x : 0.f;
          const float w1 = j + 1 <= i ? G[half][2 * e + 1] * expf((hi_i - hj.y) + (lo_i - lj.y)) * d.y : 0.f;
          uint32_t hi, lo;
          split_bf16x2(w0, w1, hi, lo);
          *reinterpret_cast<uint32_t*>(m_hi + i * SM::LDP + j) = hi;
          *reinterpret_cast<uint32_t*>(m_lo + i * SM::LDP + j) = lo;
        }
      }
    } else if (warp == 15 && more) {
      const float2 now = steps;
      steps = chunk_steps(a, t0 + 2 * CH_L, t_end, h, lane);
      chunk_sums(&sums[(c + 1) & 1], now, t_end - t0 - CH_L, bias, A, fixed, lane);
    }
    // weighted inputs: eight values per thread
    {
      const int j = threadIdx.x >> 3, p = (threadIdx.x & 7) * 8;
      float v[8];
      ld8(sx + j * SM::LDP + p, v);
      const float w = sm.last[j];
      uint4 hi, lo;
      split_bf16x2(v[0] * w, v[1] * w, hi.x, lo.x);
      split_bf16x2(v[2] * w, v[3] * w, hi.y, lo.y);
      split_bf16x2(v[4] * w, v[5] * w, hi.z, lo.z);
      split_bf16x2(v[6] * w, v[7] * w, hi.w, lo.w);
      *reinterpret_cast<uint4*>(w_hi + j * SM::LDP + p) = hi;
      *reinterpret_cast<uint4*>(w_lo + j * SM::LDP + p) = lo;
    }
    // C S: tokens 16 wr.. of the chunk, vdim quarter wq; the two terms of the state in chains of their own
    float Y[2][4] = {}, Z[2][4] = {};
#pragma unroll
    for (int k = 0; k < NP; k += 16) {
      uint32_t fc[4], fh[4], fl[4];
      const int o = 16 * wq * SM::LDN + k + frag_b(lane, SM::LDN);
      ldmatrix_x4(fc, smem_u32(sc + 16 * wr * SM::LDN + k + frag_a(lane, SM::LDN)));
      ldmatrix_x4(fh, smem_u32(s_hi + o));
      ldmatrix_x4(fl, smem_u32(s_lo + o));
      mma_bf16(Y[0], fc, fh[0], fh[1]);
      mma_bf16(Y[1], fc, fh[2], fh[3]);
      mma_bf16(Z[0], fc, fl[0], fl[1]);
      mma_bf16(Z[1], fc, fl[2], fl[3]);
    }
    const int i0 = 16 * wr + q4, i1 = i0 + 8;
    const float e0 = expf(sm.hi[i0] + sm.lo[i0]), e1 = expf(sm.hi[i1] + sm.lo[i1]);
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      Y[k][0] = (Y[k][0] + Z[k][0]) * e0;
      Y[k][1] = (Y[k][1] + Z[k][1]) * e0;
      Y[k][2] = (Y[k][2] + Z[k][2]) * e1;
      Y[k][3] = (Y[k][3] + Z[k][3]) * e1;
    }
    __syncthreads();

    // ---- phase 2: weighted scores times x, skip, store ----
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {
      if (kt > wr) continue;
      uint32_t ah[4], al[4], fx[4];
      const int o = 16 * wr * SM::LDP + 16 * kt + frag_a(lane, SM::LDP);
      ldmatrix_x4(ah, smem_u32(m_hi + o));
      ldmatrix_x4(al, smem_u32(m_lo + o));
      ldmatrix_x4_trans(fx, smem_u32(sx + 16 * kt * SM::LDP + 16 * wq + frag_b_t(lane, SM::LDP)));
      mma_bf16(Y[0], ah, fx[0], fx[1]);
      mma_bf16(Y[1], ah, fx[2], fx[3]);
      mma_bf16(Y[0], al, fx[0], fx[1]);
      mma_bf16(Y[1], al, fx[2], fx[3]);
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int i = e ? i1 : i0;
      if (i < n_tok) {
        __nv_bfloat16* yr = a.y + static_cast<long long>(t0 + i) * a.ldy + off_x;
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          const int p = 16 * wq + 8 * k + q2;
          if (p < p_valid) {
            const float2 x = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(sx + i * SM::LDP + p));
            *reinterpret_cast<uint32_t*>(yr + p) = pack_bf16x2(fmaf(D, x.x, Y[k][2 * e]), fmaf(D, x.y, Y[k][2 * e + 1]));
          }
        }
      }
    }
    // ---- state: rows 16 wr.. of vdim, state quarter wq ----
    const float keep = expf(sm.hi[CH_L - 1] + sm.lo[CH_L - 1]);
#pragma unroll
    for (int k = 0; k < NT; ++k)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[k][e] *= keep;
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {
      uint32_t ah[4], al[4];
      const int o = 16 * kt * SM::LDP + 16 * wr + frag_a_t(lane, SM::LDP);
      ldmatrix_x4_trans(ah, smem_u32(w_hi + o));
      ldmatrix_x4_trans(al, smem_u32(w_lo + o));
#pragma unroll
      for (int k = 0; k < NT; k += 2) {
        uint32_t fb[4];
        ldmatrix_x4_trans(fb, smem_u32(sb + 16 * kt * SM::LDN + wq * (NP / 4) + 8 * k + frag_b_t(lane, SM::LDN)));
        mma_bf16(S[k], ah, fb[0], fb[1]);
        mma_bf16(S[k + 1], ah, fb[2], fb[3]);
        mma_bf16(S[k], al, fb[0], fb[1]);
        mma_bf16(S[k + 1], al, fb[2], fb[3]);
      }
    }
    if (SM::BUFS == 1 && more) {
      __syncthreads();
      chunk_load<NP>(a, stage, t0 + CH_L, min(CH_L, t_end - t0 - CH_L), off_x, p_valid, off_b, off_c);
    }
  }
#pragma unroll
  for (int k = 0; k < NT; ++k)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int p = 16 * wr + q4 + (e >> 1) * 8, n = wq * (NP / 4) + 8 * k + q2 + (e & 1);
      if (p < p_valid && n < a.N) st[static_cast<long long>(p) * a.N + n] = S[k][e];
    }
}

template <int NP>
static int launch_chunk(const ChunkArgs& a, int n_seqs, cudaStream_t stream) {
  using SM = ChunkSmem<NP>;
  static thread_local int configured_dev = -1;
  int dev = 0;
  cudaGetDevice(&dev);
  if (configured_dev != dev) {
    const cudaError_t e = cudaFuncSetAttribute(ssd_chunk_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, SM::BYTES);
    if (e != cudaSuccess) {
      set_last_error("ssd_chunk: cudaFuncSetAttribute(smem=%d) failed: %s", SM::BYTES, cudaGetErrorString(e));
      return 1;
    }
    configured_dev = dev;
  }
  const dim3 grid(n_seqs, a.heads, (a.vdim + CH_P - 1) / CH_P);
  ssd_chunk_kernel<NP><<<grid, CH_THREADS, SM::BYTES, stream>>>(a);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) {
    set_last_error("ssd_chunk launch failed: %s", cudaGetErrorString(e));
    return 1;
  }
  return 0;
}

int launch_ssd_chunk_tc(const void* xbc, long long ldx, int T, const void* dt, long long ldt, const void* dt_bias,
                        const void* A_log, const void* D, const float* decay, float* state, void* y, long long ldy,
                        const int* seqs, int n_seqs, const int* cu_q, const int* kv_lens, const int* slots, int heads,
                        int vdim, int N, int groups, uint32_t* status, cudaStream_t stream);

static int chunk_dispatch(const char* what, const ChunkArgs& a, int T, int n_seqs, int form, uint32_t* status,
                          cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  if (a.groups <= 0 || a.heads % a.groups != 0 || a.vdim % 8 != 0 || a.N % 8 != 0 || a.ldx % 8 != 0 || a.ldy % 2 != 0 ||
      a.N > 256 || (reinterpret_cast<uintptr_t>(a.xbc) & 15) != 0) {
    set_last_error("%s: vdim and N (<= 256) must be multiples of 8 in 16-byte rows (vdim=%d, N=%d, ldx=%lld)", what, a.vdim,
                   a.N, a.ldx);
    return 1;
  }
  if (form == 0 && a.N <= 128 && a.ldy % 8 == 0 && (reinterpret_cast<uintptr_t>(a.y) & 15) == 0)
    return launch_ssd_chunk_tc(a.xbc, a.ldx, T, a.dt, a.ldt, a.dt_bias, a.A_log, a.D, a.decay, a.state, a.y, a.ldy, a.seqs,
                               n_seqs, a.cu_q, a.kv_lens, a.slots, a.heads, a.vdim, a.N, a.groups, status, stream);
  if (a.N <= 64) return launch_chunk<64>(a, n_seqs, stream);
  if (a.N <= 128) return launch_chunk<128>(a, n_seqs, stream);
  return launch_chunk<256>(a, n_seqs, stream);
}

}  // namespace tw

using namespace tw;

// xbc [T, ...]; form 0: tcgen05 (ssd_chunk_tc.cu) for states of up to 128 dimensions, this file's kernel otherwise;
// form 1: this file's kernel.
extern "C" int tw_ssd_chunk(const void* xbc, long long ldx, int T, const void* dt, long long ldt, const void* dt_bias,
                            const void* A_log, const void* D, float* state, void* y, long long ldy, const int* seqs,
                            int n_seqs, const int* cu_q, const int* kv_lens, const int* slots, int heads, int vdim, int N,
                            int groups, int form, uint32_t* status, cudaStream_t stream) {
  using bf = __nv_bfloat16;
  const ChunkArgs a{reinterpret_cast<const bf*>(xbc), ldx, reinterpret_cast<const bf*>(dt), ldt,
                    reinterpret_cast<const bf*>(dt_bias), reinterpret_cast<const bf*>(A_log),
                    reinterpret_cast<const bf*>(D), nullptr, state, reinterpret_cast<bf*>(y), ldy, seqs, cu_q, kv_lens,
                    slots, heads, vdim, N, groups};
  return chunk_dispatch("ssd_chunk", a, T, n_seqs, form, status, stream);
}

// The same with unit steps, a given decay per head and no skip; vkq rows are [values | keys | queries] of all heads.
extern "C" int tw_decay_chunk(const void* vkq, long long ldx, int T, const float* decay, float* state, void* y,
                              long long ldy, const int* seqs, int n_seqs, const int* cu_q, const int* kv_lens,
                              const int* slots, int heads, int vdim, int N, int form, uint32_t* status,
                              cudaStream_t stream) {
  using bf = __nv_bfloat16;
  const ChunkArgs a{reinterpret_cast<const bf*>(vkq), ldx, nullptr, 0, nullptr, nullptr, nullptr, decay, state,
                    reinterpret_cast<bf*>(y), ldy, seqs, cu_q, kv_lens, slots, heads, vdim, N, heads};
  return chunk_dispatch("decay_chunk", a, T, n_seqs, form, status, stream);
}
