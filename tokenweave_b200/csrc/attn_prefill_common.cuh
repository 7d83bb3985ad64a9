// Shared definitions of the prefill attention kernels (attn_prefill.cu, attn_prefill_split.cu).
#pragma once

#include "tw_common.cuh"

namespace tw {

constexpr int ATT_BM = 128;      // query rows per CTA
constexpr int ATT_BN = 128;      // keys per tile
constexpr int ATT_SOFTMAX_THREADS = 256;
constexpr int ATT_THREADS = 64 + ATT_SOFTMAX_THREADS;
constexpr int ATT_HALF_BYTES = 128 * 128;  // a [128 rows x 64 bf16] swizzled half tile

// 2^x with the PTX approximation ex2.approx.ftz.f32: inputs here are <= 8 or -inf, so neither exp2f()'s full range
// nor subnormal results are needed.
__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__device__ __forceinline__ float fast_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// D[tmem] (+)= A[tmem] * B[smem]: the A operand (bf16 pairs, one 32-bit column per two K elements, one
// lane per row) comes from tensor memory.
__device__ __forceinline__ void umma_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t b_desc, uint32_t idesc,
                                        uint32_t accumulate) {
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t"
      "}\n"
      ::"r"(d_tmem), "r"(a_tmem), "l"(b_desc), "r"(idesc), "r"(accumulate)
      : "memory");
}
__device__ __forceinline__ void tmem_st_32x2(uint32_t taddr, uint32_t a, uint32_t b) {
  asm volatile("tcgen05.st.sync.aligned.32x32b.x2.b32 [%0], {%1, %2};" ::"r"(taddr), "r"(a), "r"(b) : "memory");
}
__device__ __forceinline__ void tmem_ld_32x2(uint32_t taddr, uint32_t& a, uint32_t& b) {
  asm volatile("tcgen05.ld.sync.aligned.32x32b.x2.b32 {%0, %1}, [%2];" : "=r"(a), "=r"(b) : "r"(taddr) : "memory");
}

// Waits for loads from tensor memory; the registers of one that is waited for pass through, so that nothing that reads them
// moves in front.
__device__ __forceinline__ void tmem_wait_ld_of(uint32_t (&r)[32]) {
  asm volatile("tcgen05.wait::ld.sync.aligned;"
               : "+r"(r[0]), "+r"(r[1]), "+r"(r[2]), "+r"(r[3]), "+r"(r[4]), "+r"(r[5]), "+r"(r[6]), "+r"(r[7]), "+r"(r[8]),
                 "+r"(r[9]), "+r"(r[10]), "+r"(r[11]), "+r"(r[12]), "+r"(r[13]), "+r"(r[14]), "+r"(r[15]), "+r"(r[16]),
                 "+r"(r[17]), "+r"(r[18]), "+r"(r[19]), "+r"(r[20]), "+r"(r[21]), "+r"(r[22]), "+r"(r[23]), "+r"(r[24]),
                 "+r"(r[25]), "+r"(r[26]), "+r"(r[27]), "+r"(r[28]), "+r"(r[29]), "+r"(r[30]), "+r"(r[31])
               :
               : "memory");
}

// Three-input maximum and the packed two-wide fp32 forms of sm_100: half the issue slots per score.
__device__ __forceinline__ float max3f(float a, float b, float c) {
  float d;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
  return d;
}
__device__ __forceinline__ float2 fadd2(float2 a, float2 b) {
  uint64_t ra, rb, rd;
  asm("mov.b64 %0, {%1, %2};" : "=l"(ra) : "f"(a.x), "f"(a.y));
  asm("mov.b64 %0, {%1, %2};" : "=l"(rb) : "f"(b.x), "f"(b.y));
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(rd) : "l"(ra), "l"(rb));
  float2 d;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(d.x), "=f"(d.y) : "l"(rd));
  return d;
}

// e to 16 bits of mantissa in two bf16 terms: the leading one cut off (no conversion), the rest rounded
__device__ __forceinline__ void split_weights(float2 e, uint32_t& hi, uint32_t& lo) {
  const uint32_t x = __float_as_uint(e.x), y = __float_as_uint(e.y);
  hi = __byte_perm(x, y, 0x7632);
  const float2 l = fma2(make_float2(__uint_as_float(x & 0xffff0000u), __uint_as_float(y & 0xffff0000u)),
                        make_float2(-1.f, -1.f), e);
  lo = pack_bf16x2(l.x, l.y);
}

// Items of CTA `c` of `G`: round r takes the c-th item of the r-th block of G items, counted from the
// front in even rounds and from the back in odd ones (heavy items meet light ones).
__device__ __forceinline__ int split_item_index(int round, int c, int G) {
  return round * G + ((round & 1) ? (G - 1 - c) : c);
}

// The two softmax threads of a query row sit in warps w (group A) and w + 4 (group B), the same TMEM
// lane quarter; each such warp pair meets on its own named barrier (ids 1..4, 64 threads).
__device__ __forceinline__ void split_pair_sync(int quarter) {
  asm volatile("bar.sync %0, 64;" ::"r"(quarter + 1) : "memory");
}

struct AttnParams {
  __nv_bfloat16* out;
  long long ldo;
  const int* cu_q;         // [B+1] first query row of each sequence
  const int* kv_lens;      // [B] keys visible to the last query of the sequence
  const int* block_table;  // [B, max_blocks]
  const int* tile_seq;     // [num_tiles] sequence of each query tile
  const int* tile_q0;      // [num_tiles] first query (within the sequence) of the tile
  int max_blocks;
  int page;                // tokens per cache page
  int hq, hkv;
  int ring;                // head-pair kernel: K/V tile slots in use
  float scale_log2;        // softmax scale * log2(e)
  int window;              // sliding window: a query at position p sees keys (p - window, p]; 0 = unlimited
  float softcap;           // logits soft cap: s -> cap * tanh(s / cap) on the scaled scores; 0 = off
  float scale;             // softmax scale (needed with the soft cap)
  // grouped attention with its own value size (attn_prefill_split.cu only)
  int vdim;                // value columns that are stored (a multiple of 8)
  const float* slopes;     // [hq]: slope * distance is taken off the scaled score; null: off
  int sink;                // one is added to the softmax's denominator
  float out_scale;         // factor on the result
  int keep;                // keys that stay visible before a sliding window: the first `keep`
  // sigmoid form
  const float* key_bias;   // [hq]: a key counts with sigmoid(scaled score + bias), nothing is normalized; null: softmax
  int chunk;               // a query sees the keys of its own chunk of that many positions; 0: all
  const __nv_bfloat16* gate;   // [rows, hq], row stride ldg: the result is multiplied by its sigmoid; null: off
  long long ldg;
  uint32_t* status;
};

// Kernel of attn_prefill_split.cu: persistent CTAs, one query head per work item, the item's key range
// split between the two softmax groups. max_ctas bounds the grid (0 = every SM).
int launch_prefill_grouped(int D, int DV, const CUtensorMap& tmQ, const CUtensorMap& tmK, const CUtensorMap& tmV,
                           const AttnParams& p, int num_tiles, cudaStream_t stream);
int launch_prefill_split(int D, const CUtensorMap& tmQ, const CUtensorMap& tmK, const CUtensorMap& tmV,
                         const AttnParams& p, int num_tiles, int max_ctas, cudaStream_t stream);

}  // namespace tw
