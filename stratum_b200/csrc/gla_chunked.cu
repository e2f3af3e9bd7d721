// Retention over prompts: the recurrence of gla.cu with a constant decay c per head, chunk by chunk of tokens on tensor
// cores instead of token by token.  With S the state in front of a chunk of n tokens, i and j its tokens from 0 on:
//
//   o_i = c^(i + 1) q_i S + sum over j <= i of c^(i - j) (q_i . k_j) v_j          (times q_scale)
//   S  <- c^n S + sum_j k_j (c^(n - 1 - j) v_j)^T
//
// The state stays in float32 registers from the first chunk to the last.  q, k and v, which are projections, enter the
// products in two bfloat16 parts (x = hi + lo to 16 bits of mantissa, where a projection need not have more than
// bfloat16's 8); everything behind them is as wide as float32: the scores with their decays, the decayed values and the
// state go to the tensor cores in three parts (24 bits), and all products of parts that reach a float32 sum's last place
// are formed, with float32 sums: the products of the high parts in one accumulator, the small ones in another, and both
// joined to what came before by ordinary additions (the tensor cores cut their sums off instead of rounding them).  With
// `silu_qkv` q, k and v are taken through silu before they are split.
//
// A CTA owns (sequence, head, 32 columns of S).  The next chunk's q, k and v are copied to a staging buffer
// (cp.async) while one is worked on; a chunk's phases, each a barrier apart: split into parts; scores; outputs from
// scores and state; state.  Nothing depends on the other sequences of a step, and on how a sequence's tokens are cut into
// steps only in the rounding of its sums.
#include <math.h>

#include "common.cuh"
#include "gla.h"
#include "mma_common.cuh"

#define GC_COLS 32            // columns of S (of v) per CTA
#define GC_VP 40              // bfloat16 per row of v and S in shared memory: 32 + 8 of padding

__device__ __forceinline__ void gc_ldsm4(uint32_t (&a)[4], const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(a[0]), "=r"(a[1]), "=r"(a[2]), "=r"(a[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)) : "memory");
}
__device__ __forceinline__ void gc_ldsm4_t(uint32_t (&a)[4], const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(a[0]), "=r"(a[1]), "=r"(a[2]), "=r"(a[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)) : "memory");
}
__device__ __forceinline__ void gc_ldsm2(uint32_t (&b)[2], const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];"
               : "=r"(b[0]), "=r"(b[1]) : "r"((uint32_t)__cvta_generic_to_shared(p)) : "memory");
}
__device__ __forceinline__ void gc_ldsm2_t(uint32_t (&b)[2], const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];"
               : "=r"(b[0]), "=r"(b[1]) : "r"((uint32_t)__cvta_generic_to_shared(p)) : "memory");
}
__device__ __forceinline__ void gc_mma(float (&acc)[4], const uint32_t (&a)[4], const uint32_t (&b)[2]) {
  mma16816(acc, a[0], a[1], a[2], a[3], b[0], b[1]);
}
__device__ __forceinline__ void gc_split2(float x, float y, bf16* hi, bf16* lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  *reinterpret_cast<__nv_bfloat162*>(hi) = h;
  *reinterpret_cast<uint32_t*>(lo) = pack_bf16(x - __bfloat162float(h.x), y - __bfloat162float(h.y));
}
// three parts, `step` values apart: 24 bits of mantissa together
__device__ __forceinline__ void gc_split3(float x, float y, bf16* p, int step) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  x -= __bfloat162float(h.x);
  y -= __bfloat162float(h.y);
  *reinterpret_cast<__nv_bfloat162*>(p) = h;
  gc_split2(x, y, p + step, p + 2 * step);
}
__device__ __forceinline__ void gc_split4(float4 v, bf16* hi, bf16* lo) {
  gc_split2(v.x, v.y, hi, lo);
  gc_split2(v.z, v.w, hi + 2, lo + 2);
}
__device__ __forceinline__ void gc_copy16(float* dst_shared, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst_shared)), "l"(src)
               : "memory");
}

__device__ __forceinline__ float gc_silu(float z) { return __fdividef(z, 1.0f + __expf(-z)); }
__device__ __forceinline__ float4 gc_silu(float4 v) { return make_float4(gc_silu(v.x), gc_silu(v.y), gc_silu(v.z), gc_silu(v.w)); }

// Floats and bfloat16 of shared memory for chunks of C tokens and `dim` key dimensions, in this order.
__host__ __device__ __forceinline__ size_t gc_smem_bytes(int C, int dim) {
  const size_t floats = (size_t)C * (2 * dim + GC_COLS) + C + 4;                       // staging, powers of the decay
  const size_t halves = 4 * (size_t)C * (dim + 8) + 3 * (size_t)C * (C + 8) + 5 * (size_t)C * GC_VP + 3 * (size_t)dim * GC_VP;
  return floats * 4 + halves * 2;
}

// C: tokens of a chunk (64 or 32).  MB: blocks of 16 rows of S a warp holds (dim <= 128 MB): eight warps cover the rows, and
// with sixteen the other eight take the other half of the columns.
template <int C, int MB, int WARPS, bool SILU>
__global__ void __launch_bounds__(WARPS * 32) gla_chunked_kernel(const Gla P) {
  extern __shared__ __align__(16) float gc_smem[];
  constexpr int RB = C / 16;                          // blocks of 16 tokens
  constexpr int CW = WARPS / RB;                   // warps that share a block of tokens
  constexpr int NA = C / 8 / CW;                      // blocks of 8 scores a warp takes
  constexpr int NO = GC_COLS / 8 / CW;                // blocks of 8 columns of the output a warp takes
  constexpr int NS = GC_COLS / 8 / (WARPS / 8);       // blocks of 8 columns of the state a warp holds
  constexpr int AP = C + 8;                           // bfloat16 per row of the scores
  const int D = P.dim, V = P.vdim, HD = P.n_heads * D, HV = P.n_heads * V, QP = D + 8;
  float* stage_q = gc_smem;                           // [C][D]
  float* stage_k = stage_q + C * D;                   // [C][D]
  float* stage_v = stage_k + C * D;                   // [C][GC_COLS]
  float* power = stage_v + C * GC_COLS;               // [C + 1]: c^m
  bf16* q_hi = reinterpret_cast<bf16*>(power + C + 4);
  bf16* q_lo = q_hi + C * QP;
  bf16* k_hi = q_lo + C * QP;
  bf16* k_lo = k_hi + C * QP;
  const int A1 = C * AP, W1 = C * GC_VP, S1 = D * GC_VP;        // from a part of the scores, values, state to the next
  bf16* a_p = k_lo + C * QP;                          // [3][C][AP]
  bf16* v_hi = a_p + 3 * A1;                          // [C][GC_VP]
  bf16* v_lo = v_hi + W1;
  bf16* w_p = v_lo + W1;                              // [3][C][GC_VP]: v_j c^(n - 1 - j)
  bf16* s_p = w_p + 3 * W1;                           // [3][D][GC_VP]

  const int seq = blockIdx.z, h = blockIdx.y, j0 = blockIdx.x * GC_COLS;
  const int r0 = P.seq_start[seq], r1 = P.seq_start[seq + 1];
  if (r0 >= r1) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  if (P.token_seq[r0] < 0) {                          // rows of no sequence: nothing is kept, the output is zero
    for (int i = threadIdx.x; i < (r1 - r0) * GC_COLS; i += blockDim.x) {
      const int r = r0 + i / GC_COLS, j = j0 + i % GC_COLS;
      if (j < V) P.o_raw[(size_t)r * HV + (size_t)h * V + j] = 0.f;
    }
    return;
  }
  const float decay = P.head_decay[h];
  for (int m = threadIdx.x; m <= C; m += blockDim.x) power[m] = powf(decay, (float)m);
  // what this warp holds of S: blocks of 16 rows from 16 (srow + 8 b) on, NS blocks of 8 columns from scol on
  const int srow = warp % 8, scol = 8 * NS * (warp / 8);
  float* Sg = P.state + (size_t)P.seq_slot[seq] * P.state_stride + ((size_t)h * V + j0) * D;
  float S[MB][NS][4];
#pragma unroll
  for (int b = 0; b < MB; b++)
#pragma unroll
    for (int n = 0; n < NS; n++)
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const int d = 16 * (srow + 8 * b) + g + 8 * (e >> 1), j = scol + 8 * n + 2 * t + (e & 1);
        S[b][n][e] = (d < D && j0 + j < V) ? Sg[(size_t)j * D + d] : 0.f;
      }
  auto put_state = [&]() {                            // S in two parts, for the products of the next chunk
#pragma unroll
    for (int b = 0; b < MB; b++) {
      const int d = 16 * (srow + 8 * b) + g;
      if (16 * (srow + 8 * b) >= D) continue;
#pragma unroll
      for (int n = 0; n < NS; n++) {
        const int at = d * GC_VP + scol + 8 * n + 2 * t;
        gc_split3(S[b][n][0], S[b][n][1], s_p + at, S1);
        gc_split3(S[b][n][2], S[b][n][3], s_p + at + 8 * GC_VP, S1);
      }
    }
  };
  put_state();
  auto stage = [&](int c0) {                          // ask for the tokens c0 .. of this sequence; rows beyond it are zero
    const int n = min(C, r1 - c0);
    for (int tok = warp; tok < C; tok += WARPS)
     for (int d = 4 * lane; d < D; d += 128) {
      float *dq = stage_q + tok * D + d, *dk = stage_k + tok * D + d;
      if (tok < n) {
        const float* row = P.proj + (size_t)(c0 + tok) * P.ld + (size_t)h * D + d;
        gc_copy16(dq, row);
        gc_copy16(dk, row + HD);
      } else {
        *reinterpret_cast<float4*>(dq) = *reinterpret_cast<float4*>(dk) = make_float4(0.f, 0.f, 0.f, 0.f);
      }
    }
    for (int i = threadIdx.x; i < C * (GC_COLS / 4); i += blockDim.x) {
      const int tok = i / (GC_COLS / 4), j = 4 * (i % (GC_COLS / 4));
      float* dv = stage_v + tok * GC_COLS + j;
      if (tok < n && j0 + j < V) gc_copy16(dv, P.proj + (size_t)(c0 + tok) * P.ld + 2 * (size_t)HD + (size_t)h * V + j0 + j);
      else *reinterpret_cast<float4*>(dv) = make_float4(0.f, 0.f, 0.f, 0.f);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  stage(r0);
  const int rb = warp % RB, cw = warp / RB;           // this warp's block of tokens and its share of the columns
  for (int c0 = r0; c0 < r1; c0 += C) {
    const int n_here = min(C, r1 - c0);
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();                                  // the chunk has landed; the parts of the one before are free
    {
      for (int tok = warp; tok < C; tok += WARPS)
       for (int d = 4 * lane; d < D; d += 128) {
        float4 q = *reinterpret_cast<const float4*>(stage_q + tok * D + d), k = *reinterpret_cast<const float4*>(stage_k + tok * D + d);
        if (SILU) { q = gc_silu(q); k = gc_silu(k); }
        gc_split4(q, q_hi + tok * QP + d, q_lo + tok * QP + d);
        gc_split4(k, k_hi + tok * QP + d, k_lo + tok * QP + d);
      }
      for (int i = threadIdx.x; i < C * (GC_COLS / 4); i += blockDim.x) {
        const int tok = i / (GC_COLS / 4), j = 4 * (i % (GC_COLS / 4)), at = tok * GC_VP + j;
        float4 v = *reinterpret_cast<const float4*>(stage_v + tok * GC_COLS + j);
        if (SILU) v = gc_silu(v);
        gc_split4(v, v_hi + at, v_lo + at);
        const float w = tok < n_here ? power[n_here - 1 - tok] : 0.f;
        v.x *= w; v.y *= w; v.z *= w; v.w *= w;
        gc_split3(v.x, v.y, w_p + at, W1);
        gc_split3(v.z, v.w, w_p + at + 2, W1);
      }
    }
    __syncthreads();                                  // the parts are there and the staging buffer is free
    if (c0 + C < r1) stage(c0 + C);

    // ---- scores of 16 tokens against C / CW keys, decayed; what lies ahead of a token is zero
    {
      float acc[NA][4], rest[NA][4];
#pragma unroll
      for (int n = 0; n < NA; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) acc[n][e] = rest[n][e] = 0.f;
      const int first = cw * NA;                      // this warp's first block of 8 keys
      if (8 * first <= 16 * rb + 15) {
        for (int d = 0; d < D; d += 16) {
          uint32_t ah[4], al[4];
          const int at = (16 * rb + (lane & 15)) * QP + d + 8 * (lane >> 4);
          gc_ldsm4(ah, q_hi + at);
          gc_ldsm4(al, q_lo + at);
#pragma unroll
          for (int n = 0; n < NA; n++) {
            uint32_t bh[2], bl[2];
            const int bt = (8 * (first + n) + (lane & 7)) * QP + d + 8 * ((lane >> 3) & 1);
            gc_ldsm2(bh, k_hi + bt);
            gc_ldsm2(bl, k_lo + bt);
            gc_mma(acc[n], ah, bh);
            gc_mma(rest[n], al, bl);
            gc_mma(rest[n], al, bh);
            gc_mma(rest[n], ah, bl);
          }
        }
      }
#pragma unroll
      for (int n = 0; n < NA; n++) {
        const int j = 8 * (first + n) + 2 * t;
#pragma unroll
        for (int e = 0; e < 2; e++) {
          const int i = 16 * rb + g + 8 * e;
          const float x = j <= i ? (acc[n][2 * e] + rest[n][2 * e]) * power[i - j] : 0.f;
          const float y = j + 1 <= i ? (acc[n][2 * e + 1] + rest[n][2 * e + 1]) * power[i - j - 1] : 0.f;
          gc_split3(x, y, a_p + i * AP + j, A1);
        }
      }
    }
    __syncthreads();
    // ---- outputs of 16 tokens, NO blocks of 8 columns
    {
      float acc[NO][4], rest[NO][4], sum[NO][4];
#pragma unroll
      for (int n = 0; n < NO; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) acc[n][e] = rest[n][e] = 0.f;
      for (int d = 0; d < D; d += 16) {
        uint32_t ah[4], al[4];
        const int at = (16 * rb + (lane & 15)) * QP + d + 8 * (lane >> 4);
        gc_ldsm4(ah, q_hi + at);
        gc_ldsm4(al, q_lo + at);
#pragma unroll
        for (int n = 0; n < NO; n++) {
          uint32_t b0[2], b1[2], b2[2];
          const int bt = (d + (lane & 15)) * GC_VP + 8 * (cw * NO + n);
          gc_ldsm2_t(b0, s_p + bt);
          gc_ldsm2_t(b1, s_p + S1 + bt);
          gc_ldsm2_t(b2, s_p + 2 * S1 + bt);
          gc_mma(acc[n], ah, b0);
          gc_mma(rest[n], ah, b2);
          gc_mma(rest[n], al, b1);
          gc_mma(rest[n], ah, b1);
          gc_mma(rest[n], al, b0);
        }
      }
      const float p0 = power[16 * rb + g + 1], p1 = power[16 * rb + g + 9];
#pragma unroll
      for (int n = 0; n < NO; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
          sum[n][e] = (acc[n][e] + rest[n][e]) * (e < 2 ? p0 : p1);
          acc[n][e] = rest[n][e] = 0.f;
        }
#pragma unroll
      for (int kb = 0; kb < RB; kb++) {
        if (kb > rb) break;                           // keys ahead of the whole block of tokens
        uint32_t a0[4], a1[4], a2[4];
        const int at = (16 * rb + (lane & 15)) * AP + 16 * kb + 8 * (lane >> 4);
        gc_ldsm4(a0, a_p + at);
        gc_ldsm4(a1, a_p + A1 + at);
        gc_ldsm4(a2, a_p + 2 * A1 + at);
#pragma unroll
        for (int n = 0; n < NO; n++) {
          uint32_t bh[2], bl[2];
          const int bt = (16 * kb + (lane & 15)) * GC_VP + 8 * (cw * NO + n);
          gc_ldsm2_t(bh, v_hi + bt);
          gc_ldsm2_t(bl, v_lo + bt);
          gc_mma(acc[n], a0, bh);
          gc_mma(rest[n], a2, bh);
          gc_mma(rest[n], a1, bl);
          gc_mma(rest[n], a1, bh);
          gc_mma(rest[n], a0, bl);
        }
      }
#pragma unroll
      for (int n = 0; n < NO; n++) {
        const int j = j0 + 8 * (cw * NO + n) + 2 * t;
        if (j >= V) continue;                         // vdim is even: a pair of columns is inside or outside together
#pragma unroll
        for (int e = 0; e < 2; e++) {
          const int i = 16 * rb + g + 8 * e;
          if (i < n_here)
            *reinterpret_cast<float2*>(P.o_raw + (size_t)(c0 + i) * HV + (size_t)h * V + j) =
                make_float2((sum[n][2 * e] + (acc[n][2 * e] + rest[n][2 * e])) * P.q_scale,
                            (sum[n][2 * e + 1] + (acc[n][2 * e + 1] + rest[n][2 * e + 1])) * P.q_scale);
        }
      }
    }
    // ---- the state: 16 MB rows a warp
    {
      const float pn = power[n_here];
#pragma unroll
      for (int b = 0; b < MB; b++) {
        const int d0 = 16 * (srow + 8 * b);
        if (d0 >= D) continue;
        float acc[NS][4], rest[NS][4];
#pragma unroll
        for (int n = 0; n < NS; n++)
#pragma unroll
          for (int e = 0; e < 4; e++) acc[n][e] = rest[n][e] = 0.f;
#pragma unroll
        for (int kb = 0; kb < RB; kb++) {
          uint32_t ah[4], al[4];
          const int at = (16 * kb + (lane & 7) + 8 * (lane >> 4)) * QP + d0 + 8 * ((lane >> 3) & 1);
          gc_ldsm4_t(ah, k_hi + at);
          gc_ldsm4_t(al, k_lo + at);
#pragma unroll
          for (int n = 0; n < NS; n++) {
            uint32_t b0[2], b1[2], b2[2];
            const int bt = (16 * kb + (lane & 15)) * GC_VP + scol + 8 * n;
            gc_ldsm2_t(b0, w_p + bt);
            gc_ldsm2_t(b1, w_p + W1 + bt);
            gc_ldsm2_t(b2, w_p + 2 * W1 + bt);
            gc_mma(acc[n], ah, b0);
            gc_mma(rest[n], ah, b2);
            gc_mma(rest[n], al, b1);
            gc_mma(rest[n], ah, b1);
            gc_mma(rest[n], al, b0);
          }
        }
#pragma unroll
        for (int n = 0; n < NS; n++)
#pragma unroll
          for (int e = 0; e < 4; e++) S[b][n][e] = fmaf(S[b][n][e], pn, acc[n][e] + rest[n][e]);
      }
    }
    __syncthreads();                                  // every warp has read the old state
    put_state();
  }
  if (P.write_state) {
#pragma unroll
    for (int b = 0; b < MB; b++)
#pragma unroll
      for (int n = 0; n < NS; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
          const int d = 16 * (srow + 8 * b) + g + 8 * (e >> 1), j = scol + 8 * n + 2 * t + (e & 1);
          if (d < D && j0 + j < V) Sg[(size_t)j * D + d] = S[b][n][e];
        }
  }
}

template <int C, int MB, int WARPS, bool SILU>
static int gla_chunked_launch(const Gla& P, cudaStream_t stream) {
  const size_t smem = gc_smem_bytes(C, P.dim);
  if (smem > 227 * 1024) return STRATUM_ERR_LIMIT;
  cudaError_t e = cudaFuncSetAttribute(gla_chunked_kernel<C, MB, WARPS, SILU>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  const dim3 grid((P.vdim + GC_COLS - 1) / GC_COLS, P.n_heads, P.n_seqs);
  gla_chunked_kernel<C, MB, WARPS, SILU><<<grid, WARPS * 32, smem, stream>>>(P);
  return launch_status();
}

// The recurrence of a step with a constant decay per head.  Needs dim % 16 == 0, dim <= 256, vdim % 4 == 0, rows of the
// projection 16-byte aligned.
STRATUM_EXPORT int stratum_gla_chunked(const Gla* params, cudaStream_t stream) {
  const Gla& P = *params;
  if (P.n_tokens <= 0 || P.n_seqs <= 0) return 0;
  const int bad = gla_check(P);
  if (bad) return bad;
  if (!P.head_decay || P.dim % 16 != 0 || P.vdim % 4 != 0 || P.ld % 4 != 0) return STRATUM_ERR_SHAPE;
  if (((uintptr_t)P.proj & 15) != 0 || ((uintptr_t)P.o_raw & 7) != 0) return STRATUM_ERR_ALIGN;
  if (P.dim <= 128) return P.silu_qkv ? gla_chunked_launch<64, 1, 16, true>(P, stream) : gla_chunked_launch<64, 1, 16, false>(P, stream);
  if (P.dim <= 256) return P.silu_qkv ? gla_chunked_launch<32, 2, 8, true>(P, stream) : gla_chunked_launch<32, 2, 8, false>(P, stream);
  return STRATUM_ERR_LIMIT;
}
