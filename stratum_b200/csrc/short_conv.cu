// Between the query/key/value projection and attention, for mixers whose queries, keys and values pass a short causal
// convolution over time and are then neither normalised nor rotated.
//
// Per token of a sequence, from the float32 sums of the projection (row u = [q: n_heads * dim | k: n_kv * dim | v: n_kv *
// v_dim], biases in it), channel by channel:
//   y = sum_j w[j] u(t - taps + 1 + j)          inputs before the sequence's start are zero; taps = 0: y = u
//   values      with v_first_in: y <- (1 - lambda) y + lambda v_first_in[t] (an earlier layer's values of the same token);
//               with v_first_out: y also goes there, for later layers
//   q goes to q_out [tokens][ldq], k and v are appended to the paged caches, all in the compute dtype.
// Everything between the projection's sums and the rounding of the results is float32.
//
// A sequence keeps the inputs u of its last taps - 1 tokens, oldest first: state [slot][taps - 1][channels], float32, zero
// in a fresh slot.  A thread owns a few channels of a run of consecutive tokens of one sequence.  The runs of a step cut
// a sequence's tokens from its first on, and a run that is not its sequence's last one has at least taps - 1 tokens: so
// only a sequence's first run reads the state, and the thread that has read a channel's state moves it on.  A sum's order
// is the taps' order, whatever the cut.
// Rows of no sequence (sequence -1) have no past, and leave caches and states alone.
#include "common.cuh"

struct ShortConv {
  const float* proj;        // [tokens][ld]
  const float* conv_w;      // [taps][channels]
  const float* lambda;      // one number, with v_first_in
  const void* v_first_in;   // [tokens][ld_first] or null
  void* v_first_out;        // [tokens][ld_first] or null
  void* q_out;              // [tokens][ldq]
  void* k_cache;            // [pages][n_kv][page_tokens][dim]
  void* v_cache;            // [pages][n_kv][page_tokens][v_dim]
  float* state;             // [slots][state_stride]
  const int* token_pos;
  const int* token_seq;
  const int* block_table;   // [seqs][bt_stride]
  const int* run_seq;       // runs: sequence, first row, tokens; null: every row is a run of its own
  const int* run_row;
  const int* run_n;
  const int* seq_start;     // [seqs + 1]
  const int* seq_slot;      // [seqs]
  int ld, ldq, ld_first, bt_stride, n_tokens, n_runs;
  int n_heads, n_kv, dim, v_dim;
  int page_tokens, write_cache, taps, state_stride;
};

#define SC_THREADS 128
#define SC_BATCH 4            // tokens of a run whose loads are in flight together

template <int VEC> struct ScPack { float v[VEC]; };

template <int VEC>
__device__ __forceinline__ ScPack<VEC> sc_load(const float* p) {
  ScPack<VEC> r;
  if constexpr (VEC == 4) {
    const float4 x = ld_fresh(reinterpret_cast<const float4*>(p));
    r.v[0] = x.x; r.v[1] = x.y; r.v[2] = x.z; r.v[3] = x.w;
  } else {
    r.v[0] = ld_fresh(p);
  }
  return r;
}
template <int VEC>
__device__ __forceinline__ ScPack<VEC> sc_load(const bf16* p) {
  ScPack<VEC> r;
  if constexpr (VEC == 4) {
    const uint2 x = __ldcg(reinterpret_cast<const uint2*>(p));
    const __nv_bfloat162 lo = *reinterpret_cast<const __nv_bfloat162*>(&x.x), hi = *reinterpret_cast<const __nv_bfloat162*>(&x.y);
    r.v[0] = __low2float(lo); r.v[1] = __high2float(lo); r.v[2] = __low2float(hi); r.v[3] = __high2float(hi);
  } else {
    r.v[0] = ld_fresh(p);
  }
  return r;
}
template <int VEC>
__device__ __forceinline__ void sc_store(float* p, const ScPack<VEC>& r) {
  if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
  else *p = r.v[0];
}
template <int VEC>
__device__ __forceinline__ void sc_store(bf16* p, const ScPack<VEC>& r) {
  if constexpr (VEC == 4) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(r.v[0], r.v[1]), hi = __floats2bfloat162_rn(r.v[2], r.v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
  } else {
    *p = __float2bfloat16_rn(r.v[0]);
  }
}

// TAPS > 0: that many, the inputs a run shares stay in registers.  TAPS = 0: any number, every input is loaded again.
template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(SC_THREADS) short_conv_kernel(const ShortConv P) {
  pdl_trigger();
  const int nq = P.n_heads * P.dim, nk = P.n_kv * P.dim, nv = P.n_kv * P.v_dim, channels = nq + nk + nv;
  const int c = VEC * (blockIdx.y * SC_THREADS + threadIdx.x);
  const int run = blockIdx.x;
  const int row0 = P.run_row ? P.run_row[run] : run;
  const int seq = P.run_seq ? P.run_seq[run] : P.token_seq[row0];
  const int n = P.run_n ? P.run_n[run] : 1;
  const int taps = TAPS > 0 ? TAPS : P.taps;
  const int start = seq >= 0 ? P.seq_start[seq] : row0, len = seq >= 0 ? P.seq_start[seq + 1] - start : 1;
  const int in_step = row0 - start;                  // tokens of the sequence in front of this run, in this step
  if (c >= channels) return;
  float* st = taps > 1 && seq >= 0 ? P.state + (size_t)P.seq_slot[seq] * P.state_stride + c : nullptr;
  const float* in = P.proj + (size_t)row0 * P.ld + c;
  // where the channels go: q 0, k 1, v 2, and the column within
  const int part = c < nq ? 0 : (c < nq + nk ? 1 : 2);
  const int col = part == 0 ? c : (part == 1 ? c - nq : c - nq - nk);
  const int size = part == 2 ? P.v_dim : P.dim;
  const int head = col / size, d = col - head * size;
  ScPack<VEC> w[TAPS > 0 ? TAPS : 1], hist[TAPS > 1 ? TAPS - 1 : 1];
#pragma unroll
  for (int j = 0; j < TAPS; j++)
#pragma unroll
    for (int e = 0; e < VEC; e++) w[j].v[e] = P.conv_w[(size_t)j * channels + c + e];
  const bool writes = P.write_cache && seq >= 0;
  const int* bt = writes && part > 0 ? P.block_table + (size_t)seq * P.bt_stride : nullptr;
  const int pos0 = P.token_pos[row0];
  int page_of = pos0 / P.page_tokens, page = bt ? bt[page_of] : -1;      // the page looked up last
  pdl_wait();              // the projection, the state and the first values are the work of kernels before this one
  if (n <= 0) return;      // an entry of a list of fixed length that holds no token
  // the input `back` tokens in front of row i of the run
  auto input = [&](int i, int back) -> ScPack<VEC> {
    if (back <= in_step + i) return sc_load<VEC>(in + ((long long)i - back) * P.ld);
    if (st) return sc_load<VEC>(st + (size_t)(taps - 1 + in_step + i - back) * channels);
    ScPack<VEC> zero;
#pragma unroll
    for (int e = 0; e < VEC; e++) zero.v[e] = 0.f;
    return zero;
  };
  if (TAPS > 1) {
#pragma unroll
    for (int j = 0; j < TAPS - 1; j++) hist[j] = input(0, TAPS - 1 - j);
  }
  const float lam = part == 2 && P.v_first_in ? *P.lambda : 0.f;
  for (int i0 = 0; i0 < n; i0 += SC_BATCH) {
    // a batch's loads go out together
    ScPack<VEC> u[SC_BATCH], first[SC_BATCH];
    if (TAPS > 0 || taps == 0) {
#pragma unroll
      for (int b = 0; b < SC_BATCH; b++)
        if (i0 + b < n) u[b] = sc_load<VEC>(in + (size_t)(i0 + b) * P.ld);
    }
    if (part == 2 && P.v_first_in) {
#pragma unroll
      for (int b = 0; b < SC_BATCH; b++)
        if (i0 + b < n) first[b] = sc_load<VEC>((const T*)P.v_first_in + (size_t)(row0 + i0 + b) * P.ld_first + col);
    }
#pragma unroll
    for (int b = 0; b < SC_BATCH; b++) {
      const int i = i0 + b;
      if (i >= n) break;
      ScPack<VEC> y;
      if (TAPS > 0) {
#pragma unroll
        for (int e = 0; e < VEC; e++) {
          float acc = 0.f;
#pragma unroll
          for (int j = 0; j < TAPS - 1; j++) acc = fmaf(w[j].v[e], hist[j].v[e], acc);      // oldest input first
          y.v[e] = fmaf(w[TAPS > 0 ? TAPS - 1 : 0].v[e], u[b].v[e], acc);
        }
#pragma unroll
        for (int j = 0; j + 1 < TAPS - 1; j++) hist[j] = hist[j + 1];
        if (TAPS > 1) hist[TAPS > 1 ? TAPS - 2 : 0] = u[b];
      } else if (taps == 0) {
        y = u[b];
      } else {
#pragma unroll
        for (int e = 0; e < VEC; e++) y.v[e] = 0.f;
        for (int j = 0; j < taps; j++) {
          const ScPack<VEC> x = input(i, taps - 1 - j);
#pragma unroll
          for (int e = 0; e < VEC; e++) y.v[e] = fmaf(P.conv_w[(size_t)j * channels + c + e], x.v[e], y.v[e]);
        }
      }
      const size_t row = (size_t)(row0 + i);
      if (part == 0) {
        sc_store<VEC>((T*)P.q_out + row * P.ldq + col, y);
        continue;
      }
      if (part == 2) {
        if (P.v_first_in) {
#pragma unroll
          for (int e = 0; e < VEC; e++) y.v[e] = (1.0f - lam) * y.v[e] + lam * first[b].v[e];
        }
        if (P.v_first_out) sc_store<VEC>((T*)P.v_first_out + row * P.ld_first + col, y);
      }
      if (!writes) continue;
      const int pos = pos0 + i, nth = pos / P.page_tokens;
      if (nth != page_of) { page_of = nth; page = bt[nth]; }
      if (page < 0) continue;
      T* cache = (T*)(part == 1 ? P.k_cache : P.v_cache);
      sc_store<VEC>(cache + (((size_t)page * P.n_kv + head) * P.page_tokens + (pos - nth * P.page_tokens)) * size + d, y);
    }
  }
  // the sequence's first run moves its state on: row r becomes what stands `len` places further in (state, then the
  // step's tokens); rows are read ahead of where they are written
  if (P.write_cache && st && in_step == 0) {
    for (int r = 0; r < taps - 1; r++) {
      const int from = r + len - (taps - 1);
      const ScPack<VEC> u = from >= 0 ? sc_load<VEC>(in + (size_t)from * P.ld) : sc_load<VEC>(st + (size_t)(r + len) * channels);
      sc_store<VEC>(st + (size_t)r * channels, u);
    }
  }
}

template <typename T>
static int short_conv_launch(const ShortConv& P, int vec, cudaStream_t stream) {
  const int channels = P.n_heads * P.dim + P.n_kv * (P.dim + P.v_dim), per = SC_THREADS * (vec ? 4 : 1);
  const dim3 grid((unsigned)P.n_runs, (unsigned)((channels + per - 1) / per));
  if (!vec) return launch_pdl(short_conv_kernel<T, 1, 0>, grid, SC_THREADS, 0, stream, P);
  switch (P.taps) {
    case 1: return launch_pdl(short_conv_kernel<T, 4, 1>, grid, SC_THREADS, 0, stream, P);
    case 2: return launch_pdl(short_conv_kernel<T, 4, 2>, grid, SC_THREADS, 0, stream, P);
    case 3: return launch_pdl(short_conv_kernel<T, 4, 3>, grid, SC_THREADS, 0, stream, P);
    case 4: return launch_pdl(short_conv_kernel<T, 4, 4>, grid, SC_THREADS, 0, stream, P);
    default: return launch_pdl(short_conv_kernel<T, 4, 0>, grid, SC_THREADS, 0, stream, P);
  }
}

STRATUM_EXPORT int stratum_short_conv(const ShortConv* params, int dtype, cudaStream_t stream) {
  const ShortConv& P = *params;
  if (P.n_tokens <= 0 || P.n_runs <= 0) return 0;
  if (P.n_heads < 1 || P.n_kv < 1 || P.dim < 1 || P.v_dim < 1 || P.taps < 0 || P.page_tokens < 1) return STRATUM_ERR_SHAPE;
  const int nq = P.n_heads * P.dim, nv = P.n_kv * P.v_dim, channels = nq + P.n_kv * P.dim + nv;
  if (P.ld < channels || P.ldq < nq || !P.seq_start || (P.taps > 0 && !P.conv_w)) return STRATUM_ERR_SHAPE;
  if (P.taps > 1 && (!P.state || !P.seq_slot || P.state_stride < (P.taps - 1) * channels)) return STRATUM_ERR_SHAPE;
  if ((P.v_first_in || P.v_first_out) && P.ld_first < nv) return STRATUM_ERR_SHAPE;
  if (P.v_first_in && !P.lambda) return STRATUM_ERR_SHAPE;
  if (P.write_cache && (!P.k_cache || !P.v_cache || !P.block_table)) return STRATUM_ERR_SHAPE;
  if (channels > 65535 * SC_THREADS) return STRATUM_ERR_LIMIT;
  if (dtype != STRATUM_DT_F32 && dtype != STRATUM_DT_BF16) return STRATUM_ERR_DTYPE;
  const int vec = P.dim % 4 == 0 && P.v_dim % 4 == 0 && P.ld % 4 == 0 && P.ldq % 4 == 0 && P.ld_first % 4 == 0 &&
                  P.state_stride % 4 == 0 &&
                  (((uintptr_t)P.proj | (uintptr_t)P.v_first_in | (uintptr_t)P.v_first_out | (uintptr_t)P.q_out |
                    (uintptr_t)P.k_cache | (uintptr_t)P.v_cache | (uintptr_t)P.state) & 15) == 0;
  return dtype == STRATUM_DT_F32 ? short_conv_launch<float>(P, vec, stream) : short_conv_launch<bf16>(P, vec, stream);
}
