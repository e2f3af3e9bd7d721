// Between the query/key(/value) projection and attention, for mixers whose queries and keys are RMS-normalised
// before they are rotated.
//
// Per token, from the float32 sums of the projection (row = [q: n_heads * dim | k: n_kv * dim | v: n_kv * v_dim]):
//   values   v_dim = 0: the key columns as projected; else the value columns; rounded once to the cache's dtype and
//            appended to the value cache;
//   q, k     divided by a root mean square (eps inside the root) and multiplied by a gain: of the whole stretch (all
//            heads together) with a gain per column, or (per_head) of every head by itself with one gain of `dim`
//            values for all heads; then in every head the first 2 * rot_pairs dimensions are turned by the angle
//            pos * inv_freq[i] (float32), (u, v) -> ((u cos - v sin) m, (v cos + u sin) m) with m the magnitude:
//            pairs (2i, 2i + 1), or (half) pairs (i, i + rot_pairs);
//   q goes to q_out [tokens][ldq] in the compute dtype, k is appended to the key cache.
// Everything between the projection's sums and the rounding of the results is float32.  Tokens of no sequence
// (sequence index -1) write nothing to the caches.  One block per token; the block's shape is fixed, so a row's sums
// do not depend on the step.
// Rows in multiples of four values (16-byte aligned) take a form that reads the row once, into shared memory, as vectors,
// and evaluates every angle of the token once.
#include <math.h>

#include "common.cuh"

struct QKNormRope {
  const float* proj;        // [tokens][ld]
  const int* token_pos;
  const int* token_seq;
  const int* block_table;   // [seqs][bt_stride]
  const float* q_gain;      // [n_heads * dim]
  const float* k_gain;      // [n_kv * dim]
  const float* inv_freq;    // [rot_pairs]
  void* q_out;              // [tokens][ldq]
  void* k_cache;            // [pages][n_kv][page_tokens][dim]
  void* v_cache;            // the same shape, or [pages][n_kv][page_tokens][v_dim]
  int ld, ldq, bt_stride, n_tokens;
  int n_heads, n_kv, dim, rot_pairs;
  int page_tokens, write_cache;
  float eps, magnitude;
  int v_dim, per_head, half, reserved;
};

#define QK_THREADS 256

// the value of column c (of a stretch that begins at column c0 of the row) after norm and rotation
__device__ __forceinline__ float qk_turned(const QKNormRope& P, const float* row, int c0, int c, int d, float mul,
                                           const float* gain, int pos) {
  const int g = P.per_head ? d : c;
  float v = ld_fresh(row + c0 + c) * mul * gain[g];
  const int rp = P.rot_pairs;
  if (d < 2 * rp) {
    int mate, pair;
    bool second;
    if (P.half) { second = d >= rp; mate = second ? c - rp : c + rp; pair = second ? d - rp : d; }
    else { second = d & 1; mate = second ? c - 1 : c + 1; pair = d >> 1; }
    const float w = ld_fresh(row + c0 + mate) * mul * gain[P.per_head ? d + (mate - c) : mate];
    float sn, cs;
    sincosf((float)pos * P.inv_freq[pair], &sn, &cs);
    v = (second ? v * cs + w * sn : v * cs - w * sn) * P.magnitude;
  }
  return v;
}

template <typename T>
__global__ void __launch_bounds__(QK_THREADS) qk_norm_rope_kernel(const QKNormRope P) {
  __shared__ float scratch[33];
  extern __shared__ float head_mul[];                // per_head: 1 / rms of every query head, then of every key head
  pdl_trigger();
  pdl_wait();                                        // the projection is the work of the kernel before: ld_fresh
  const int t = blockIdx.x;
  const float* row = P.proj + (size_t)t * P.ld;
  const int D = P.dim, nq = P.n_heads * D, nk = P.n_kv * D;
  float sq = 0.f, sk = 0.f;
  if (P.per_head) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int h = warp; h < P.n_heads + P.n_kv; h += QK_THREADS / 32) {     // a head's sum: one warp, one order
      float ss = 0.f;
      for (int d = lane; d < D; d += 32) {
        const float v = ld_fresh(row + (size_t)h * D + d);
        ss = fmaf(v, v, ss);
      }
      ss = warp_sum(ss);
      if (lane == 0) head_mul[h] = 1.0f / sqrtf(ss / (float)D + P.eps);
    }
    __syncthreads();
  } else {
    float ssq = 0.f, ssk = 0.f;
    for (int c = threadIdx.x; c < nq; c += QK_THREADS) {
      const float v = ld_fresh(row + c);
      ssq = fmaf(v, v, ssq);
    }
    for (int c = threadIdx.x; c < nk; c += QK_THREADS) {
      const float v = ld_fresh(row + nq + c);
      ssk = fmaf(v, v, ssk);
    }
    ssq = block_sum(ssq, scratch);
    ssk = block_sum(ssk, scratch);
    sq = 1.0f / sqrtf(ssq / (float)nq + P.eps);
    sk = 1.0f / sqrtf(ssk / (float)nk + P.eps);
  }
  const int pos = P.token_pos[t], seq = P.token_seq[t];

  T* qo = (T*)P.q_out + (size_t)t * P.ldq;
  for (int c = threadIdx.x; c < nq; c += QK_THREADS) {
    const int h = c / D, d = c - h * D;
    qo[c] = from_float<T>(qk_turned(P, row, 0, c, d, P.per_head ? head_mul[h] : sq, P.q_gain, pos));
  }
  if (!P.write_cache || seq < 0) return;
  const int page = P.block_table[(size_t)seq * P.bt_stride + pos / P.page_tokens];
  if (page < 0) return;
  const int in_page = pos % P.page_tokens;
  for (int c = threadIdx.x; c < nk; c += QK_THREADS) {
    const int h = c / D, d = c - h * D;
    const size_t at = (((size_t)page * P.n_kv + h) * P.page_tokens + in_page) * D + d;
    if (P.v_dim == 0) ((T*)P.v_cache)[at] = from_float<T>(ld_fresh(row + nq + c));
    ((T*)P.k_cache)[at] =
        from_float<T>(qk_turned(P, row, nq, c, d, P.per_head ? head_mul[P.n_heads + h] : sk, P.k_gain, pos));
  }
  const int V = P.v_dim;
  for (int c = threadIdx.x; c < P.n_kv * V; c += QK_THREADS) {
    const int h = c / V, d = c - h * V;
    const size_t at = (((size_t)page * P.n_kv + h) * P.page_tokens + in_page) * V + d;
    ((T*)P.v_cache)[at] = from_float<T>(ld_fresh(row + nq + nk + c));
  }
}

// The form for rows in multiples of four values.
#define QK_ROW_THREADS 256
__device__ __forceinline__ void qk_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void qk_store4(bf16* p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<const uint32_t*>(&a);
  u.y = *reinterpret_cast<const uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = u;
}

template <typename T>
__global__ void __launch_bounds__(QK_ROW_THREADS) qk_norm_rope_row_kernel(const QKNormRope P) {
  extern __shared__ __align__(16) float qk_row[];    // the row's queries and keys | cos, sin | 1 / rms per head
  __shared__ float sums[2][QK_ROW_THREADS / 32];
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int D = P.dim, nq = P.n_heads * D, nk = P.n_kv * D, nv = P.n_kv * P.v_dim, heads = P.n_heads + P.n_kv;
  float2* cs = reinterpret_cast<float2*>(qk_row + nq + nk);
  float* mul = reinterpret_cast<float*>(cs + P.rot_pairs);
  pdl_trigger();
  const int pos = P.token_pos[t], seq = P.token_seq[t];
  for (int i = threadIdx.x; i < P.rot_pairs; i += QK_ROW_THREADS) {
    float sn, c;
    sincosf((float)pos * P.inv_freq[i], &sn, &c);
    cs[i] = make_float2(c, sn);
  }
  const int page = P.write_cache && seq >= 0 ? P.block_table[(size_t)seq * P.bt_stride + pos / P.page_tokens] : -1;
  const int in_page = pos % P.page_tokens;
  const float* row = P.proj + (size_t)t * P.ld;
  pdl_wait();                                        // the projection is the work of the kernel before: ld_fresh
  float ssq = 0.f, ssk = 0.f;
  for (int c = 4 * threadIdx.x; c < nq + nk; c += 4 * QK_ROW_THREADS) {
    const float4 v = ld_fresh(reinterpret_cast<const float4*>(row + c));
    *reinterpret_cast<float4*>(qk_row + c) = v;
    const float s = fmaf(v.w, v.w, fmaf(v.z, v.z, fmaf(v.y, v.y, v.x * v.x)));
    if (c < nq) ssq += s; else ssk += s;
  }
  if (page >= 0) {                                   // values: no norm, no rotation
    for (int c = 4 * threadIdx.x; c < nv; c += 4 * QK_ROW_THREADS) {
      const int h = c / P.v_dim, d = c - h * P.v_dim;
      qk_store4((T*)P.v_cache + (((size_t)page * P.n_kv + h) * P.page_tokens + in_page) * P.v_dim + d,
                ld_fresh(reinterpret_cast<const float4*>(row + nq + nk + c)));
    }
  }
  if (P.per_head) {
    __syncthreads();
    for (int h = warp; h < heads; h += QK_ROW_THREADS / 32) {          // a head's sum: one warp, one order
      float ss = 0.f;
      for (int d = lane; d < D; d += 32) ss = fmaf(qk_row[h * D + d], qk_row[h * D + d], ss);
      ss = warp_sum(ss);
      if (lane == 0) mul[h] = 1.0f / sqrtf(ss / (float)D + P.eps);
    }
    __syncthreads();
  } else {
    ssq = warp_sum(ssq);
    ssk = warp_sum(ssk);
    if (lane == 0) { sums[0][warp] = ssq; sums[1][warp] = ssk; }
    __syncthreads();
    ssq = ssk = 0.f;
#pragma unroll
    for (int w = 0; w < QK_ROW_THREADS / 32; w++) { ssq += sums[0][w]; ssk += sums[1][w]; }
    ssq = 1.0f / sqrtf(ssq / (float)nq + P.eps);
    ssk = 1.0f / sqrtf(ssk / (float)nk + P.eps);
  }
  T* qo = (T*)P.q_out + (size_t)t * P.ldq;
  const int rp = P.rot_pairs, last = page >= 0 ? nq + nk : nq;
  for (int c = 4 * threadIdx.x; c < last; c += 4 * QK_ROW_THREADS) {
    const bool is_q = c < nq;
    const int h = c / D, d0 = c - h * D;             // heads of queries, then of keys
    const float m = P.per_head ? mul[h] : (is_q ? ssq : ssk);
    const float* gain = is_q ? P.q_gain : P.k_gain;
    const int g0 = P.per_head ? d0 : (is_q ? c : c - nq);
    const float4 own = *reinterpret_cast<const float4*>(qk_row + c), og = *reinterpret_cast<const float4*>(gain + g0);
    float out[4] = {own.x * m * og.x, own.y * m * og.y, own.z * m * og.z, own.w * m * og.w};
    if (d0 < 2 * rp) {
      if (P.half) {                                  // (rot_pairs is a multiple of four: four dimensions turn alike)
        const bool second = d0 >= rp;
        const int step = second ? -rp : rp, pair = second ? d0 - rp : d0;
        const float4 w = *reinterpret_cast<const float4*>(qk_row + c + step);
        const float4 wg = *reinterpret_cast<const float4*>(gain + g0 + step);
        const float4 f0 = *reinterpret_cast<const float4*>(cs + pair), f1 = *reinterpret_cast<const float4*>(cs + pair + 2);
        const float mate[4] = {w.x * m * wg.x, w.y * m * wg.y, w.z * m * wg.z, w.w * m * wg.w};
        const float cc[4] = {f0.x, f0.z, f1.x, f1.z}, ss[4] = {f0.y, f0.w, f1.y, f1.w};
#pragma unroll
        for (int i = 0; i < 4; i++)
          out[i] = (second ? out[i] * cc[i] + mate[i] * ss[i] : out[i] * cc[i] - mate[i] * ss[i]) * P.magnitude;
      } else {
#pragma unroll
        for (int i = 0; i < 4; i += 2) {
          if (d0 + i < 2 * rp) {
            const float2 f = cs[(d0 + i) >> 1];
            const float u = out[i], v = out[i + 1];
            out[i] = (u * f.x - v * f.y) * P.magnitude;
            out[i + 1] = (v * f.x + u * f.y) * P.magnitude;
          }
        }
      }
    }
    const float4 v4 = make_float4(out[0], out[1], out[2], out[3]);
    if (is_q) {
      qk_store4(qo + c, v4);
    } else {
      const size_t at = (((size_t)page * P.n_kv + h - P.n_heads) * P.page_tokens + in_page) * D + d0;
      qk_store4((T*)P.k_cache + at, v4);
      if (P.v_dim == 0) qk_store4((T*)P.v_cache + at, *reinterpret_cast<const float4*>(qk_row + c));
    }
  }
}

STRATUM_EXPORT int stratum_qk_norm_rope(const QKNormRope* params, int dtype, cudaStream_t stream) {
  const QKNormRope& P = *params;
  if (P.n_tokens <= 0) return 0;
  if (P.n_heads < 1 || P.n_kv < 1 || P.dim < 1 || P.rot_pairs < 0 || 2 * P.rot_pairs > P.dim || P.page_tokens < 1)
    return STRATUM_ERR_SHAPE;
  if (P.v_dim < 0 || P.ld < (P.n_heads + P.n_kv) * P.dim + P.n_kv * P.v_dim || P.ldq < P.n_heads * P.dim)
    return STRATUM_ERR_SHAPE;
  const size_t smem = P.per_head ? (size_t)(P.n_heads + P.n_kv) * sizeof(float) : 0;
  if (smem > 40 * 1024) return STRATUM_ERR_LIMIT;
  // (which form: by sizes and alignment alone, which a model's buffers share from step to step)
  const uintptr_t bits = (uintptr_t)P.proj | (uintptr_t)P.q_out | (uintptr_t)P.k_cache | (uintptr_t)P.v_cache |
                         (uintptr_t)P.q_gain | (uintptr_t)P.k_gain;
  const size_t row_smem = ((size_t)(P.n_heads + P.n_kv) * (P.dim + 1) + 2 * (size_t)P.rot_pairs) * sizeof(float);
  if (P.dim % 4 == 0 && (!P.half || P.rot_pairs % 4 == 0) && P.v_dim % 4 == 0 && P.ld % 4 == 0 && P.ldq % 4 == 0 && (bits & 15) == 0 && row_smem <= 100 * 1024 &&
      (dtype == STRATUM_DT_F32 || dtype == STRATUM_DT_BF16)) {
    void (*kern)(const QKNormRope) = dtype == STRATUM_DT_F32 ? qk_norm_rope_row_kernel<float> : qk_norm_rope_row_kernel<bf16>;
    if (row_smem > 40 * 1024) {
      cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)row_smem);
      if (e != cudaSuccess) return (int)e;
    }
    launch_pdl(kern, P.n_tokens, QK_ROW_THREADS, row_smem, stream, P);
    return launch_status();
  }
  if (dtype == STRATUM_DT_F32) launch_pdl(qk_norm_rope_kernel<float>, P.n_tokens, QK_THREADS, smem, stream, P);
  else if (dtype == STRATUM_DT_BF16) launch_pdl(qk_norm_rope_kernel<bf16>, P.n_tokens, QK_THREADS, smem, stream, P);
  else return STRATUM_ERR_DTYPE;
  return launch_status();
}
