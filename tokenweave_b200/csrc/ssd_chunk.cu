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
// One CTA (eight warps) per sequence, head and 64 rows of vdim. The state lives in accumulator registers for the
// whole sequence and passes through shared memory once per chunk as the operand of C S; the next chunk's B, C and x
// arrive by cp.async meanwhile.
#include "tw_host.h"
#include "tw_kernels.h"
#include "tw_mma.cuh"
#include "tw_typed.cuh"

namespace tw {

struct ChunkArgs {
  const __nv_bfloat16* xbc; long long ldx;       // [T, heads * vdim | groups * N | groups * N]
  const __nv_bfloat16* dt; long long ldt;        // [T, heads]
  const __nv_bfloat16 *dt_bias, *A_log, *D;      // [heads]
  float* state;                                  // [slots, heads, vdim, N]
  __nv_bfloat16* y; long long ldy;
  const int *seqs, *cu_q, *kv_lens, *slots;
  int heads, vdim, N, groups;
};

constexpr int CH_L = 64;          // tokens per chunk
constexpr int CH_P = 64;          // rows of vdim per CTA
constexpr int CH_THREADS = 256;

template <int NP>
struct ChunkSmem {
  static constexpr int BUFS = NP <= 128 ? 2 : 1;
  static constexpr int LDN = NP + 8, LDP = CH_P + 8;           // padded rows: conflict-free ldmatrix
  static constexpr int BC = CH_L * LDN, X = CH_L * LDP;        // elements
  static constexpr int STAGE = 2 * BC + X;
  static constexpr int S_ELEMS = CH_P * LDN;
  static constexpr int BYTES = (BUFS * STAGE + 2 * S_ELEMS) * 2 + 2 * 4 * CH_L * 4;
};

// Running sums of one chunk by one warp: token 2 lane and 2 lane + 1 per lane.
struct ChunkSums {
  float dt[CH_L];      // step sizes, zero behind the run's end
  float hi[CH_L], lo[CH_L];
  float last[CH_L];    // exp(l_last - l_j) dt_j
};

__device__ __forceinline__ void chunk_sums(const ChunkArgs& a, ChunkSums* s, int t0, int n, int h, float bias, float A,
                                           int lane) {
  double l[2];
  float d[2];
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int j = 2 * lane + e;
    d[e] = j < n ? softplus_f(ld1(a.dt + (t0 + j) * a.ldt + h) + bias) : 0.f;
    l[e] = -static_cast<double>(A) * d[e];
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
  constexpr int NT = NP / 16;                // 8-column tiles of this warp's half of the state dimension
  extern __shared__ __align__(16) uint8_t smem_raw[];
  __nv_bfloat16* stage = reinterpret_cast<__nv_bfloat16*>(smem_raw);
  __nv_bfloat16* s_hi = stage + SM::BUFS * SM::STAGE;
  __nv_bfloat16* s_lo = s_hi + SM::S_ELEMS;
  ChunkSums* sums = reinterpret_cast<ChunkSums*>(s_lo + SM::S_ELEMS);     // [2]

  const int b = a.seqs[blockIdx.x], h = blockIdx.y, p0 = blockIdx.z * CH_P;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int wr = warp & 3, wh = warp >> 2;   // row group (tokens for y, vdim for the state) and half of the columns
  const int q4 = lane >> 2, q2 = (lane & 3) * 2;
  const int t_begin = a.cu_q[b], t_end = a.cu_q[b + 1];
  const int p_valid = min(CH_P, a.vdim - p0);
  const int g = h / (a.heads / a.groups);
  const int off_x = h * a.vdim + p0, off_b = a.heads * a.vdim + g * a.N, off_c = off_b + a.groups * a.N;
  const float bias = ld1(a.dt_bias + h), A = expf(ld1(a.A_log + h)), D = ld1(a.D + h);

  // state rows p = 16 wr + q4 (+ 8), columns n = wh NP/2 + 8 k + q2 (+ 1)
  float S[NT][4];
  float* st = a.state + ((static_cast<long long>(a.slots[b]) * a.heads + h) * a.vdim + p0) * a.N;
  const bool past = a.kv_lens[b] > t_end - t_begin;
#pragma unroll
  for (int k = 0; k < NT; ++k)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int p = 16 * wr + q4 + (e >> 1) * 8, n = wh * (NP / 2) + 8 * k + q2 + (e & 1);
      S[k][e] = (past && p < p_valid && n < a.N) ? st[static_cast<long long>(p) * a.N + n] : 0.f;
    }

  chunk_load<NP>(a, stage, t_begin, min(CH_L, t_end - t_begin), off_x, p_valid, off_b, off_c);
  if (warp == 0) chunk_sums(a, &sums[0], t_begin, min(CH_L, t_end - t_begin), h, bias, A, lane);

  int c = 0;
  for (int t0 = t_begin; t0 < t_end; t0 += CH_L, ++c) {
    const int n_tok = min(CH_L, t_end - t0);
    __nv_bfloat16* cur = stage + (SM::BUFS == 2 ? (c & 1) : 0) * SM::STAGE;
    const __nv_bfloat16 *sb = cur, *sc = cur + SM::BC, *sx = cur + 2 * SM::BC;
    const ChunkSums& sm = sums[c & 1];
    // the state as the operand of C S
#pragma unroll
    for (int k = 0; k < NT; ++k) {
      const int n = wh * (NP / 2) + 8 * k + q2;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        uint32_t hi, lo;
        split_bf16x2(S[k][2 * e], S[k][2 * e + 1], hi, lo);
        const int o = (16 * wr + q4 + 8 * e) * SM::LDN + n;
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

    // ---- C S and C B^T: tokens 16 wr.. of the chunk, vdim half wh ----
    float Y[4][4] = {}, G[8][4] = {};
#pragma unroll
    for (int k = 0; k < NP; k += 16) {
      uint32_t fc[4];
      ldmatrix_x4(fc, smem_u32(sc + 16 * wr * SM::LDN + k + frag_a(lane, SM::LDN)));
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        uint32_t fh[4], fl[4];
        const int o = (32 * wh + 16 * i) * SM::LDN + k + frag_b(lane, SM::LDN);
        ldmatrix_x4(fh, smem_u32(s_hi + o));
        ldmatrix_x4(fl, smem_u32(s_lo + o));
        mma_bf16(Y[2 * i], fc, fh[0], fh[1]);
        mma_bf16(Y[2 * i + 1], fc, fh[2], fh[3]);
        mma_bf16(Y[2 * i], fc, fl[0], fl[1]);
        mma_bf16(Y[2 * i + 1], fc, fl[2], fl[3]);
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        if (i <= wr) {                        // keys behind the row group's last token are masked anyway
          uint32_t fb[4];
          ldmatrix_x4(fb, smem_u32(sb + 16 * i * SM::LDN + k + frag_b(lane, SM::LDN)));
          mma_bf16(G[2 * i], fc, fb[0], fb[1]);
          mma_bf16(G[2 * i + 1], fc, fb[2], fb[3]);
        }
      }
    }
    const int i0 = 16 * wr + q4, i1 = i0 + 8;
    const float h0 = sm.hi[i0], l0 = sm.lo[i0], h1 = sm.hi[i1], l1 = sm.lo[i1];
    const float e0 = expf(h0 + l0), e1 = expf(h1 + l1);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      Y[i][0] *= e0;
      Y[i][1] *= e0;
      Y[i][2] *= e1;
      Y[i][3] *= e1;
    }
    // ---- weighted scores times x ----
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {
      if (kt > wr) continue;
      uint32_t ah[4], al[4];
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        float w[4];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int j = 16 * kt + 8 * half + q2 + e;
          const float hj = sm.hi[j], lj = sm.lo[j], d = sm.dt[j];
          w[e] = j <= i0 ? G[2 * kt + half][e] * expf((h0 - hj) + (l0 - lj)) * d : 0.f;
          w[2 + e] = j <= i1 ? G[2 * kt + half][2 + e] * expf((h1 - hj) + (l1 - lj)) * d : 0.f;
        }
        split_bf16x2(w[0], w[1], ah[2 * half], al[2 * half]);
        split_bf16x2(w[2], w[3], ah[2 * half + 1], al[2 * half + 1]);
      }
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        uint32_t fx[4];
        ldmatrix_x4_trans(fx, smem_u32(sx + 16 * kt * SM::LDP + 32 * wh + 16 * i + frag_b_t(lane, SM::LDP)));
        mma_bf16(Y[2 * i], ah, fx[0], fx[1]);
        mma_bf16(Y[2 * i + 1], ah, fx[2], fx[3]);
        mma_bf16(Y[2 * i], al, fx[0], fx[1]);
        mma_bf16(Y[2 * i + 1], al, fx[2], fx[3]);
      }
    }
    // ---- skip and store ----
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int i = e ? i1 : i0;
      if (i < n_tok) {
        __nv_bfloat16* yr = a.y + static_cast<long long>(t0 + i) * a.ldy + off_x;
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const int p = 32 * wh + 8 * k + q2;
          if (p < p_valid) {
            const float2 x = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(sx + i * SM::LDP + p));
            *reinterpret_cast<uint32_t*>(yr + p) = pack_bf16x2(fmaf(D, x.x, Y[k][2 * e]), fmaf(D, x.y, Y[k][2 * e + 1]));
          }
        }
      }
    }
    // ---- state: rows 16 wr.. of vdim, state half wh ----
    const float keep = expf(sm.hi[CH_L - 1] + sm.lo[CH_L - 1]);
#pragma unroll
    for (int k = 0; k < NT; ++k)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[k][e] *= keep;
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {
      uint32_t fx[4], ah[4], al[4];
      ldmatrix_x4_trans(fx, smem_u32(sx + 16 * kt * SM::LDP + 16 * wr + frag_a_t(lane, SM::LDP)));
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        const float2 x = unpack_bf16x2(fx[r]);
        const int j = 16 * kt + (r >> 1) * 8 + q2;
        split_bf16x2(x.x * sm.last[j], x.y * sm.last[j + 1], ah[r], al[r]);
      }
#pragma unroll
      for (int k = 0; k < NT; k += 2) {
        uint32_t fb[4];
        ldmatrix_x4_trans(fb, smem_u32(sb + 16 * kt * SM::LDN + wh * (NP / 2) + 8 * k + frag_b_t(lane, SM::LDN)));
        mma_bf16(S[k], ah, fb[0], fb[1]);
        mma_bf16(S[k + 1], ah, fb[2], fb[3]);
        mma_bf16(S[k], al, fb[0], fb[1]);
        mma_bf16(S[k + 1], al, fb[2], fb[3]);
      }
    }
    if (warp == 0 && more)
      chunk_sums(a, &sums[(c + 1) & 1], t0 + CH_L, min(CH_L, t_end - t0 - CH_L), h, bias, A, lane);
    __syncthreads();
    if (SM::BUFS == 1 && more)
      chunk_load<NP>(a, stage, t0 + CH_L, min(CH_L, t_end - t0 - CH_L), off_x, p_valid, off_b, off_c);
  }
#pragma unroll
  for (int k = 0; k < NT; ++k)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int p = 16 * wr + q4 + (e >> 1) * 8, n = wh * (NP / 2) + 8 * k + q2 + (e & 1);
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

}  // namespace tw

using namespace tw;

extern "C" int tw_ssd_chunk(const void* xbc, long long ldx, const void* dt, long long ldt, const void* dt_bias,
                            const void* A_log, const void* D, float* state, void* y, long long ldy, const int* seqs,
                            int n_seqs, const int* cu_q, const int* kv_lens, const int* slots, int heads, int vdim, int N,
                            int groups, cudaStream_t stream) {
  if (n_seqs <= 0) return 0;
  if (groups <= 0 || heads % groups != 0 || vdim % 8 != 0 || N % 8 != 0 || ldx % 8 != 0 || ldy % 2 != 0 || N > 256 ||
      (reinterpret_cast<uintptr_t>(xbc) & 15) != 0) {
    set_last_error("ssd_chunk: vdim and N (<= 256) must be multiples of 8 in 16-byte rows (vdim=%d, N=%d, ldx=%lld)", vdim,
                   N, ldx);
    return 1;
  }
  using bf = __nv_bfloat16;
  const ChunkArgs a{reinterpret_cast<const bf*>(xbc), ldx, reinterpret_cast<const bf*>(dt), ldt,
                    reinterpret_cast<const bf*>(dt_bias), reinterpret_cast<const bf*>(A_log),
                    reinterpret_cast<const bf*>(D), state, reinterpret_cast<bf*>(y), ldy, seqs, cu_q, kv_lens, slots,
                    heads, vdim, N, groups};
  if (N <= 32) return launch_chunk<32>(a, n_seqs, stream);
  if (N <= 64) return launch_chunk<64>(a, n_seqs, stream);
  if (N <= 128) return launch_chunk<128>(a, n_seqs, stream);
  return launch_chunk<256>(a, n_seqs, stream);
}
