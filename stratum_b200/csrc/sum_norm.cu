// The norm of a sum: the residual stream times a constant plus up to two outputs of sublayers, each of which may first be
// divided by its row's root mean square, normalised over equal groups of the row.
//
//   z   = scale * x[row] + sum_j ( y_j[r] / sqrt(mean(y_j[r]^2) + eps_j) * gain_j   or, without a gain,   y_j[r] )
//   out = groups > 0:  z cut into `groups` equal consecutive parts, each over sqrt(mean(part^2) + eps), times gain
//         groups = 0:  z
//
// float32 in and inside; out float32 (it may be x itself) or bfloat16, and optionally a bfloat16 copy beside a float32
// one (what the next sublayer's matrix products read).  `rows` picks rows of x (the rows whose logits are wanted).
//
// One block per row.  The warps are dealt out to the groups, so that a group's sum of squares is one of few warps'; a
// thread keeps its values in registers from the loads to the stores.  The block's shape and the order of every sum
// follow from the row's length and the number of groups alone, never from how many rows a step has.
#include "common.cuh"

#define SN_TERMS 2

struct SumNorm {
  const float* x;              // [rows of the stream][hidden]
  const int* rows;             // [n_rows] or null: row r of the result comes from row r of x
  const float* y[SN_TERMS];    // [n_rows][hidden] or null
  const float* y_gain[SN_TERMS];   // [hidden] or null: the term is added as it is
  const float* gain;           // [hidden] (groups > 0)
  void* out;                   // [n_rows][hidden]
  bf16* copy;                  // [n_rows][hidden] or null
  int n_rows, hidden, groups, n_terms;
  float scale, eps, y_eps[SN_TERMS];
  int reserved;
};

__device__ __forceinline__ void sn_store(float* out, size_t i, float4 v) { *reinterpret_cast<float4*>(out + i) = v; }
__device__ __forceinline__ void sn_store(bf16* out, size_t i, float4 v) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  uint2 pk;
  pk.x = *reinterpret_cast<uint32_t*>(&lo);
  pk.y = *reinterpret_cast<uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(out + i) = pk;
}
__device__ __forceinline__ float sn_dot(float4 v) { return fmaf(v.w, v.w, fmaf(v.z, v.z, fmaf(v.y, v.y, v.x * v.x))); }
__device__ __forceinline__ void sn_axpy(float4& z, float a, float4 y, float4 g) {
  z.x = fmaf(y.x * a, g.x, z.x); z.y = fmaf(y.y * a, g.y, z.y); z.z = fmaf(y.z * a, g.z, z.z); z.w = fmaf(y.w * a, g.w, z.w);
}

// Rows whose groups are a multiple of four values, at most KEEP pieces of four per thread; `team` warps per group.
// (as many warps as the registers of KEEP pieces leave room for)
__host__ __device__ constexpr int sn_most_warps(int keep) { return keep == 2 ? 32 : 16; }

template <typename T, int KEEP>
__global__ void __launch_bounds__(sn_most_warps(KEEP) * 32) sum_norm_vec_kernel(const SumNorm P, int team) {
  __shared__ float part[SN_TERMS][32], zpart[32];
  pdl_trigger();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
  const int n_groups = P.groups > 0 ? P.groups : 1, size4 = P.hidden / n_groups / 4;
  const int group = warp / team, within = (warp - group * team) * 32 + lane;
  const int first = group * size4;                    // the group's first piece
  const int r = blockIdx.x;
  pdl_wait();                                         // x and the terms are the work of kernels before this one: ld_fresh
  const int src = P.rows ? P.rows[r] : r;
  const float4* xr = reinterpret_cast<const float4*>(P.x + (size_t)src * P.hidden);
  float4 z[KEEP], y[SN_TERMS][KEEP];
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int k = 0; k < KEEP; k++) {
    const int i = within + k * team * 32;
    const bool ok = i < size4;
    z[k] = ok && P.scale != 0.f ? ld_fresh(xr + first + i) : zero;
#pragma unroll
    for (int j = 0; j < SN_TERMS; j++)
      y[j][k] = ok && P.y[j] ? ld_fresh(reinterpret_cast<const float4*>(P.y[j] + (size_t)r * P.hidden) + first + i) : zero;
  }
  float mul[SN_TERMS] = {1.f, 1.f};
  const bool normed = P.y_gain[0] || P.y_gain[1];
  if (normed) {
#pragma unroll
    for (int j = 0; j < SN_TERMS; j++) {
      float ss = 0.f;
#pragma unroll
      for (int k = 0; k < KEEP; k++) ss += sn_dot(y[j][k]);
      ss = warp_sum(ss);
      if (lane == 0) part[j][warp] = ss;
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < SN_TERMS; j++) {
      float ss = 0.f;
      for (int w = 0; w < n_warps; w++) ss += part[j][w];
      if (P.y_gain[j]) mul[j] = 1.0f / sqrtf(ss / (float)P.hidden + P.y_eps[j]);
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < KEEP; k++) {
    const int i = within + k * team * 32;
    if (i >= size4) continue;
    float4 v = make_float4(z[k].x * P.scale, z[k].y * P.scale, z[k].z * P.scale, z[k].w * P.scale);
#pragma unroll
    for (int j = 0; j < SN_TERMS; j++) {
      const float4 g = P.y_gain[j] ? reinterpret_cast<const float4*>(P.y_gain[j])[first + i] : make_float4(1.f, 1.f, 1.f, 1.f);
      sn_axpy(v, mul[j], y[j][k], g);
    }
    z[k] = v;
    ss += sn_dot(v);
  }
  float m = 1.f;
  if (P.groups > 0) {
    ss = warp_sum(ss);
    if (lane == 0) zpart[warp] = ss;
    __syncthreads();
    float t = 0.f;
    for (int w = 0; w < team; w++) t += zpart[group * team + w];
    m = 1.0f / sqrtf(t / (float)(4 * size4) + P.eps);
  }
#pragma unroll
  for (int k = 0; k < KEEP; k++) {
    const int i = within + k * team * 32;
    if (i >= size4) continue;
    float4 v = z[k];
    if (P.groups > 0) {
      const float4 g = reinterpret_cast<const float4*>(P.gain)[first + i];
      v = make_float4(v.x * m * g.x, v.y * m * g.y, v.z * m * g.z, v.w * m * g.w);
    }
    const size_t at = (size_t)r * P.hidden + 4 * (size_t)(first + i);
    sn_store((T*)P.out, at, v);
    if (P.copy) sn_store(P.copy, at, v);
  }
}

// Any row: one value at a time, z in shared memory, the block takes one group after another.
template <typename T>
__global__ void __launch_bounds__(256) sum_norm_any_kernel(const SumNorm P) {
  extern __shared__ float sn_z[];                     // [hidden]
  __shared__ float scratch[33];
  pdl_trigger();
  const int r = blockIdx.x;
  pdl_wait();
  const int src = P.rows ? P.rows[r] : r;
  const float* xr = P.x + (size_t)src * P.hidden;
  float mul[SN_TERMS] = {1.f, 1.f};
#pragma unroll
  for (int j = 0; j < SN_TERMS; j++) {
    if (!P.y_gain[j]) continue;
    const float* yr = P.y[j] + (size_t)r * P.hidden;
    float ss = 0.f;
    for (int i = threadIdx.x; i < P.hidden; i += blockDim.x) { const float v = ld_fresh(yr + i); ss = fmaf(v, v, ss); }
    mul[j] = 1.0f / sqrtf(block_sum(ss, scratch) / (float)P.hidden + P.y_eps[j]);
  }
  for (int i = threadIdx.x; i < P.hidden; i += blockDim.x) {
    float z = P.scale != 0.f ? ld_fresh(xr + i) * P.scale : 0.f;
#pragma unroll
    for (int j = 0; j < SN_TERMS; j++)
      if (P.y[j]) z = fmaf(ld_fresh(P.y[j] + (size_t)r * P.hidden + i) * mul[j], P.y_gain[j] ? P.y_gain[j][i] : 1.f, z);
    sn_z[i] = z;
  }
  __syncthreads();
  const int n_groups = P.groups > 0 ? P.groups : 1, size = P.hidden / n_groups;
  T* out = (T*)P.out + (size_t)r * P.hidden;
  for (int g = 0; g < n_groups; g++) {
    float m = 1.f;
    if (P.groups > 0) {
      float ss = 0.f;
      for (int i = threadIdx.x; i < size; i += blockDim.x) { const float v = sn_z[g * size + i]; ss = fmaf(v, v, ss); }
      m = 1.0f / sqrtf(block_sum(ss, scratch) / (float)size + P.eps);
    }
    for (int i = g * size + threadIdx.x; i < (g + 1) * size; i += blockDim.x) {
      const float v = P.groups > 0 ? sn_z[i] * m * P.gain[i] : sn_z[i];
      out[i] = from_float<T>(v);
      if (P.copy) P.copy[(size_t)r * P.hidden + i] = __float2bfloat16_rn(v);
    }
  }
}

template <typename T>
static int launch_sum_norm(const SumNorm& P, cudaStream_t stream) {
  const int n_groups = P.groups > 0 ? P.groups : 1, size = P.hidden / n_groups;
  uintptr_t bits = (uintptr_t)P.x | (uintptr_t)P.gain | (uintptr_t)P.out | (uintptr_t)P.copy;
  for (int j = 0; j < SN_TERMS; j++) bits |= (uintptr_t)P.y[j] | (uintptr_t)P.y_gain[j];
  // (the choice depends on the row's length and on alignment alone, which a model's buffers share from step to step)
  if (size % 4 == 0 && (bits & 15) == 0 && n_groups <= 32) {
    const int pieces = size / 4;
    int keep = 0, team = 0;
    for (int k : {4, 8, 2}) {
      team = (pieces + 32 * k - 1) / (32 * k);
      if (team * n_groups <= sn_most_warps(k)) { keep = k; break; }
    }
    if (keep) {
      const dim3 block(n_groups * team * 32);
      if (keep == 2) launch_pdl(sum_norm_vec_kernel<T, 2>, P.n_rows, block, 0, stream, P, team);
      else if (keep == 4) launch_pdl(sum_norm_vec_kernel<T, 4>, P.n_rows, block, 0, stream, P, team);
      else launch_pdl(sum_norm_vec_kernel<T, 8>, P.n_rows, block, 0, stream, P, team);
      return launch_status();
    }
  }
  const size_t smem = (size_t)P.hidden * sizeof(float);
  if (smem > 200 * 1024) return STRATUM_ERR_LIMIT;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(sum_norm_any_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  launch_pdl(sum_norm_any_kernel<T>, P.n_rows, 256, smem, stream, P);
  return launch_status();
}

STRATUM_EXPORT int stratum_sum_norm(const SumNorm* params, int out_dtype, cudaStream_t stream) {
  const SumNorm& P = *params;
  if (P.n_rows <= 0) return 0;
  if (P.hidden < 1 || P.groups < 0 || (P.groups > 0 && (P.hidden % P.groups != 0 || !P.gain))) return STRATUM_ERR_SHAPE;
  for (int j = 0; j < SN_TERMS; j++)
    if (P.y_gain[j] && !P.y[j]) return STRATUM_ERR_SHAPE;
  if (out_dtype == STRATUM_DT_F32) return launch_sum_norm<float>(P, stream);
  if (out_dtype == STRATUM_DT_BF16) return launch_sum_norm<bf16>(P, stream);
  return STRATUM_ERR_DTYPE;
}
