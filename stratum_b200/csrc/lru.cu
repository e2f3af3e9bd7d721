// A gated linear recurrence (a real-gated linear recurrent unit behind a short convolution): per channel one number S.
//
// Per token, from the float32 sums of the input projection (branches y and x, `width` columns each):
//   u = conv_b + sum_j conv_w[j] x(t - taps + 1 + j)          per channel, inputs before the sequence's start are zero
//   r, i = sigmoid(A_b u_b + .), sigmoid(B_b u_b + .)         per block b of `size` neighbouring channels
//   a = exp(rate * r);  S <- a S + sqrt(1 - a^2) i u          1 - a^2 = -e (2 + e), e = expm1(rate r)
//   out = S * gelu_tanh(y)                                    rounded to the compute dtype for the output product
// All of it is float32 whatever the compute dtype; the gates' matrices may be bfloat16, and the tensor cores then take
// the float32 rows u in two bfloat16 parts (u = hi + lo to 16 bits of mantissa), with float32 sums.
//
// A sequence keeps S [width] and the last inputs of the convolution as a ring [taps][width]: the input of position p lies
// in row p % taps, so a step that brings one token writes a row that none of its own readers needs.
//
// Three kernels for prompts (conv, gates, scan) and one for decode steps (step).  The scan runs over time in parallel: a
// block owns 16 channels of a sequence, half a warp a stretch of tokens; every stretch is reduced to (product of a, end
// value from zero), the stretches are chained in shared memory, and every stretch runs its tokens again from the value it
// is handed, from registers.  Nothing depends on the other sequences of a step.
#include <math.h>

#include "common.cuh"
#include "mma_common.cuh"

struct Lru {
  const float* y;           // [tokens][ld]
  const float* x;           // [tokens][ld]
  const float* conv_w;      // [taps][width]
  const float* conv_b;      // [width]
  const void* gate_w;       // [blocks][2 size][size]: A_b's rows, then B_b's
  const float* gate_b;      // [blocks][2 size]
  const float* rate;        // [width]
  float* u;                 // [tokens][width]
  float* pre;               // [tokens][2 width]: block b's r and i before bias and sigmoid at column 2 size b
  void* out;                // [tokens][ldo]
  float* state;             // [slots][state_stride]: S [width], ring [taps][width]
  const int* token_pos;
  const int* token_seq;
  const int* seq_start;     // [seqs + 1]
  const int* seq_slot;      // [seqs]
  int ld, ldo, n_tokens, n_seqs, width, blocks, taps, state_stride, write_state, max_new;
};

// FAST: exponential and quotient of the special function unit (a few units in the last place of float32) instead of the
// library's, on the bfloat16 path.
__device__ __forceinline__ float lru_quick_reciprocal(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float lru_quick_root(float x) {
  float y;
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
template <bool FAST>
__device__ __forceinline__ float lru_sigmoid(float z) {
  return FAST ? lru_quick_reciprocal(1.0f + __expf(-z)) : 1.0f / (1.0f + expf(-z));
}
// exp(x) - 1 for x <= 0: its Taylor series to x^7 where |x| < 1/4 (what is left out is below 2^-29 of the first
// term), the exponential itself below that, where the difference costs at most three bits
__device__ __forceinline__ float lru_quick_expm1(float x) {
  float s = fmaf(x, 1.0f / 5040.0f, 1.0f / 720.0f);
  s = fmaf(s, x, 1.0f / 120.0f);
  s = fmaf(s, x, 1.0f / 24.0f);
  s = fmaf(s, x, 1.0f / 6.0f);
  s = fmaf(s, x, 0.5f);
  s = fmaf(s * x, x, x);
  return x > -0.25f ? s : __expf(x) - 1.0f;
}
template <bool FAST>
__device__ __forceinline__ float lru_gelu(float z) {   // (1 + tanh w) / 2 = sigmoid(2 w)
  if (!FAST) return activate(z, STRATUM_ACT_GELU_TANH);
  return z * lru_sigmoid<true>(1.59576912160573071176f * (z + 0.044715f * z * z * z));
}
// (a, b) of S <- a S + b.  Both from e = a - 1, which keeps its digits where a is nearly one: 1 - a^2 = -e (2 + e).
template <bool FAST>
__device__ __forceinline__ float2 lru_coefficients(float r_pre, float i_pre, float u, float rate) {
  const float la = rate * lru_sigmoid<FAST>(r_pre);
  const float e = FAST ? lru_quick_expm1(la) : expm1f(la), q = -e * (2.0f + e);
  return make_float2(1.0f + e, (FAST ? lru_quick_root(q) : sqrtf(q)) * lru_sigmoid<FAST>(i_pre) * u);
}

// ---------------------------------------------------------------- conv: a thread per (run of tokens, channel)
// TAPS > 0: the inputs a run shares stay in registers.  TAPS = 0: any number of taps, every input is loaded again.
#define LRU_RUN 8
#define LRU_CONV_THREADS 128

__device__ __forceinline__ float lru_input(const Lru& P, int t, int back, int in_step, int pos, const float* ring, int c) {
  if (back <= in_step) return ld_fresh(P.x + (size_t)(t - back) * P.ld + c);
  if (ring && pos - back >= 0) return ld_fresh(ring + (size_t)((pos - back) % P.taps) * P.width + c);
  return 0.f;
}

template <int TAPS>
__global__ void __launch_bounds__(LRU_CONV_THREADS) lru_conv_kernel(const Lru P) {
  pdl_trigger();
  pdl_wait();                // the projection and the state are the work of kernels before this one: ld_fresh
  const int c = blockIdx.y * LRU_CONV_THREADS + threadIdx.x;
  if (c >= P.width) return;
  const int t0 = blockIdx.x * LRU_RUN, t1 = min(P.n_tokens, t0 + LRU_RUN);
  const int taps = TAPS > 0 ? TAPS : P.taps;
  const float bias = P.conv_b[c];
  float w[TAPS > 0 ? TAPS : 1], hist[TAPS > 0 ? TAPS : 1];      // hist[j]: the input taps - 1 - j tokens back
#pragma unroll
  for (int j = 0; j < TAPS; j++) { w[j] = P.conv_w[(size_t)j * P.width + c]; hist[j] = 0.f; }
  for (int t = t0; t < t1; t++) {
    const int seq = P.token_seq[t];
    const int pos = P.token_pos[t];
    const int in_step = seq >= 0 ? t - P.seq_start[seq] : 0;
    const float* ring = seq >= 0 ? P.state + (size_t)P.seq_slot[seq] * P.state_stride + P.width : nullptr;
    float acc = bias;
    if (TAPS > 0) {
      if (t == t0 || in_step == 0) {
#pragma unroll
        for (int j = 0; j < TAPS - 1; j++) hist[j] = lru_input(P, t, TAPS - 1 - j, in_step, pos, ring, c);
      }
      hist[TAPS > 0 ? TAPS - 1 : 0] = ld_fresh(P.x + (size_t)t * P.ld + c);
#pragma unroll
      for (int j = 0; j < TAPS; j++) acc = fmaf(w[j], hist[j], acc);       // oldest input first: one fixed order
#pragma unroll
      for (int j = 0; j + 1 < TAPS; j++) hist[j] = hist[j + 1];
    } else {
      for (int j = 0; j < taps; j++)
        acc = fmaf(P.conv_w[(size_t)j * P.width + c], lru_input(P, t, taps - 1 - j, in_step, pos, ring, c), acc);
    }
    P.u[(size_t)t * P.width + c] = acc;
  }
}

// The same for taps that stay in registers, four channels a thread (width in multiples of four, aligned).
template <int TAPS>
__global__ void __launch_bounds__(LRU_CONV_THREADS) lru_conv_vec_kernel(const Lru P) {
  pdl_trigger();
  pdl_wait();
  const int c = 4 * (blockIdx.y * LRU_CONV_THREADS + threadIdx.x);
  if (c >= P.width) return;
  const int t0 = blockIdx.x * LRU_RUN, t1 = min(P.n_tokens, t0 + LRU_RUN);
  const float4 bias = *reinterpret_cast<const float4*>(P.conv_b + c);
  float4 w[TAPS], hist[TAPS];
#pragma unroll
  for (int j = 0; j < TAPS; j++) {
    w[j] = *reinterpret_cast<const float4*>(P.conv_w + (size_t)j * P.width + c);
    hist[j] = make_float4(0.f, 0.f, 0.f, 0.f);
  }
#pragma unroll
  for (int i = 0; i < LRU_RUN; i++) {
    const int t = t0 + i;
    if (t >= t1) break;
    const int seq = P.token_seq[t], pos = P.token_pos[t];
    const int in_step = seq >= 0 ? t - P.seq_start[seq] : 0;
    if (i == 0 || in_step == 0) {
      const float* ring = seq >= 0 ? P.state + (size_t)P.seq_slot[seq] * P.state_stride + P.width : nullptr;
#pragma unroll
      for (int j = 0; j < TAPS - 1; j++) {
        const int back = TAPS - 1 - j;
        if (back <= in_step) hist[j] = ld_fresh((const float4*)(P.x + (size_t)(t - back) * P.ld + c));
        else if (ring && pos - back >= 0) hist[j] = ld_fresh((const float4*)(ring + (size_t)((pos - back) % TAPS) * P.width + c));
        else hist[j] = make_float4(0.f, 0.f, 0.f, 0.f);
      }
    }
    hist[TAPS - 1] = ld_fresh((const float4*)(P.x + (size_t)t * P.ld + c));
    float4 u = bias;
#pragma unroll
    for (int j = 0; j < TAPS; j++) {                 // oldest input first: the order of the other form
      u.x = fmaf(w[j].x, hist[j].x, u.x); u.y = fmaf(w[j].y, hist[j].y, u.y);
      u.z = fmaf(w[j].z, hist[j].z, u.z); u.w = fmaf(w[j].w, hist[j].w, u.w);
    }
    *reinterpret_cast<float4*>(P.u + (size_t)t * P.width + c) = u;
#pragma unroll
    for (int j = 0; j + 1 < TAPS; j++) hist[j] = hist[j + 1];
  }
}

// ---------------------------------------------------------------- gates: block-diagonal product on tensor cores
// A CTA of eight warps owns 128 tokens and 128 of a block's 2 size columns; a warp 64 x 32 of them.  u is split into its
// two bfloat16 parts on the way to shared memory; the next chunk of k is on its way while one is multiplied.
#define LG_M 128
#define LG_N 128
#define LG_K 32
#define LG_PITCH 40           // bfloat16 per row in shared memory: 32 + 8 of padding (rows fall on different banks)
#define LG_STAGE (2 * LG_M * LG_PITCH + LG_N * LG_PITCH)       // hi, lo, weights

__device__ __forceinline__ void lg_ldmatrix4(uint32_t (&a)[4], const bf16* lane_row) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(a[0]), "=r"(a[1]), "=r"(a[2]), "=r"(a[3])
               : "r"((uint32_t)__cvta_generic_to_shared(lane_row)) : "memory");
}
__device__ __forceinline__ void split_bf16(float4 v, uint2& hi, uint2& lo) {
  const __nv_bfloat162 h0 = __floats2bfloat162_rn(v.x, v.y), h1 = __floats2bfloat162_rn(v.z, v.w);
  hi.x = *reinterpret_cast<const uint32_t*>(&h0);
  hi.y = *reinterpret_cast<const uint32_t*>(&h1);
  lo.x = pack_bf16(v.x - __bfloat162float(h0.x), v.y - __bfloat162float(h0.y));
  lo.y = pack_bf16(v.z - __bfloat162float(h1.x), v.w - __bfloat162float(h1.y));
}

__global__ void __launch_bounds__(256) lru_gates_kernel(const Lru P) {
  extern __shared__ __align__(16) bf16 lg_smem[];               // [2][LG_STAGE]
  const int size = P.width / P.blocks, two = 2 * size;
  const int b = blockIdx.z, m0 = blockIdx.x * LG_M, n0 = blockIdx.y * LG_N;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int wm = (warp >> 2) * 64, wn = (warp & 3) * 32;
  const bf16* wb = (const bf16*)P.gate_w + (size_t)b * two * size;
  const float* ub = P.u + (size_t)b * size;
  pdl_trigger();
  pdl_wait();

  float acc[4][4][4];
#pragma unroll
  for (int i = 0; i < 4; i++)
#pragma unroll
    for (int j = 0; j < 4; j++) { acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f; }

  // what a thread brings per chunk of k: four float4 of u (rows 32 apart), two 16-byte pieces of weights (rows 64 apart)
  const int ur = threadIdx.x >> 3, uk = (threadIdx.x & 7) * 4;
  const int wr = threadIdx.x >> 2, wk = (threadIdx.x & 3) * 8;
  float4 un[4];
  uint4 wv[2];
  auto load = [&](int k0) {
#pragma unroll
    for (int i = 0; i < 4; i++) {
      const int m = m0 + ur + 32 * i, k = k0 + uk;
      un[i] = (m < P.n_tokens && k < size) ? ld_fresh((const float4*)(ub + (size_t)m * P.width + k)) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int i = 0; i < 2; i++) {
      const int n = n0 + wr + 64 * i, k = k0 + wk;
      wv[i] = (n < two && k < size) ? __ldg((const uint4*)(wb + (size_t)n * size + k)) : make_uint4(0, 0, 0, 0);
    }
  };
  auto put = [&](int buf) {
    bf16* hi = lg_smem + buf * LG_STAGE;
    bf16* lo = hi + LG_M * LG_PITCH;
    bf16* ws = lo + LG_M * LG_PITCH;
#pragma unroll
    for (int i = 0; i < 4; i++) {
      uint2 h, l;
      split_bf16(un[i], h, l);
      *reinterpret_cast<uint2*>(hi + (ur + 32 * i) * LG_PITCH + uk) = h;
      *reinterpret_cast<uint2*>(lo + (ur + 32 * i) * LG_PITCH + uk) = l;
    }
#pragma unroll
    for (int i = 0; i < 2; i++) *reinterpret_cast<uint4*>(ws + (wr + 64 * i) * LG_PITCH + wk) = wv[i];
  };
  load(0);
  put(0);
  __syncthreads();
  int buf = 0;
  for (int k0 = 0; k0 < size; k0 += LG_K, buf ^= 1) {
    const bool more = k0 + LG_K < size;
    if (more) load(k0 + LG_K);
    const bf16* hi = lg_smem + buf * LG_STAGE;
    const bf16* lo = hi + LG_M * LG_PITCH;
    const bf16* ws = lo + LG_M * LG_PITCH;
#pragma unroll
    for (int kk = 0; kk < LG_K; kk += 16) {
      uint32_t bw[4][2];
#pragma unroll
      for (int j = 0; j < 2; j++) {        // four 8 x 8 blocks: 16 columns of the result, both halves of the 16 k
        uint32_t q[4];
        lg_ldmatrix4(q, ws + (wn + 16 * j + (lane & 7) + 8 * (lane >> 4)) * LG_PITCH + kk + 8 * ((lane >> 3) & 1));
        bw[2 * j][0] = q[0]; bw[2 * j][1] = q[1]; bw[2 * j + 1][0] = q[2]; bw[2 * j + 1][1] = q[3];
      }
#pragma unroll
      for (int i = 0; i < 4; i++) {
        uint32_t ah[4], al[4];
        const int at = (wm + 16 * i + (lane & 15)) * LG_PITCH + kk + 8 * (lane >> 4);
        lg_ldmatrix4(ah, hi + at);
        lg_ldmatrix4(al, lo + at);
#pragma unroll
        for (int j = 0; j < 4; j++) {
          mma16816(acc[i][j], ah[0], ah[1], ah[2], ah[3], bw[j][0], bw[j][1]);
          mma16816(acc[i][j], al[0], al[1], al[2], al[3], bw[j][0], bw[j][1]);
        }
      }
    }
    if (more) put(buf ^ 1);                // the other buffer was read a barrier ago
    __syncthreads();
  }
  const int g = lane >> 2, t = lane & 3;
#pragma unroll
  for (int i = 0; i < 4; i++)
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const int n = n0 + wn + 8 * j + 2 * t;
      if (n >= two) continue;              // two is even: a pair of columns is inside or outside together
#pragma unroll
      for (int e = 0; e < 2; e++) {
        const int m = m0 + wm + 16 * i + g + 8 * e;
        if (m < P.n_tokens)
          *reinterpret_cast<float2*>(P.pre + (size_t)m * 2 * P.width + (size_t)b * two + n) =
              make_float2(acc[i][j][2 * e], acc[i][j][2 * e + 1]);
      }
    }
}

// ---------------------------------------------------------------- scan
#define LS_TOKENS 8           // tokens of a stretch
#define LS_CHANNELS 16        // channels of a block: two stretches a warp
#define LS_MAX_WARPS 16

template <typename T>
__global__ void __launch_bounds__(LS_MAX_WARPS * 32, 2) lru_scan_kernel(const Lru P) {
  constexpr bool FAST = sizeof(T) == 2;
  __shared__ float2 ends[2][2 * LS_MAX_WARPS][LS_CHANNELS];      // product of a, end value from zero
  const int stretch = threadIdx.x / LS_CHANNELS, lane = threadIdx.x % LS_CHANNELS, n_stretches = blockDim.x / LS_CHANNELS;
  const int seq = blockIdx.y, c = blockIdx.x * LS_CHANNELS + lane;
  const int r0 = P.seq_start[seq], r1 = P.seq_start[seq + 1];
  if (r0 >= r1) return;
  const bool live = c < P.width;
  if (P.token_seq[r0] < 0) {                         // rows of no sequence: nothing is kept, the output is zero
    for (int r = r0 + stretch; r < r1; r += n_stretches)
      if (live) ((T*)P.out)[(size_t)r * P.ldo + c] = from_float<T>(0.f);
    return;
  }
  const int size = P.width / P.blocks, cc = live ? c : 0;
  const int col_r = (cc / size) * size + cc, col_i = col_r + size;      // 2 size b + (c - size b), then i's
  float* slot = P.state + (size_t)P.seq_slot[seq] * P.state_stride;
  const float rate = P.rate[cc], bias_r = P.gate_b[col_r], bias_i = P.gate_b[col_i];
  float S = live ? slot[cc] : 0.f;                   // the value in front of the round, the same in every stretch
  int buf = 0;
  for (int base = r0; base < r1; base += n_stretches * LS_TOKENS, buf ^= 1) {
    const int t0 = base + stretch * LS_TOKENS;
    float a[LS_TOKENS], b[LS_TOKENS], yv[LS_TOKENS];
    float uu[LS_TOKENS], rr[LS_TOKENS], ii[LS_TOKENS];
    const float* pu = P.u + (size_t)t0 * P.width + cc;
    const float* pr = P.pre + (size_t)t0 * 2 * P.width + col_r;
    const float* py = P.y + (size_t)t0 * P.ld + cc;
    float A = 1.f, H = 0.f;
    if (t0 + LS_TOKENS <= r1) {                      // a whole stretch (channels beyond the width read the first one's)
#pragma unroll
      for (int j = 0; j < LS_TOKENS; j++) {          // all loads of the stretch first
        uu[j] = pu[(size_t)(j * P.width)];
        rr[j] = pr[(size_t)(2 * j * P.width)];
        ii[j] = pr[(size_t)(2 * j * P.width) + size];
        yv[j] = py[(size_t)j * P.ld];
      }
#pragma unroll
      for (int j = 0; j < LS_TOKENS; j++) {
        const float2 ab = lru_coefficients<FAST>(rr[j] + bias_r, ii[j] + bias_i, uu[j], rate);
        a[j] = ab.x;
        b[j] = ab.y;
        A *= a[j];
        H = fmaf(a[j], H, b[j]);
      }
    } else {
#pragma unroll
      for (int j = 0; j < LS_TOKENS; j++) {
        const bool ok = t0 + j < r1;
        uu[j] = ok ? pu[(size_t)(j * P.width)] : 0.f;
        rr[j] = ok ? pr[(size_t)(2 * j * P.width)] : 0.f;
        ii[j] = ok ? pr[(size_t)(2 * j * P.width) + size] : 0.f;
        yv[j] = ok ? py[(size_t)j * P.ld] : 0.f;
        const float2 ab = lru_coefficients<FAST>(rr[j] + bias_r, ii[j] + bias_i, uu[j], rate);
        a[j] = ok ? ab.x : 1.f;
        b[j] = ok ? ab.y : 0.f;
        A *= a[j];
        H = fmaf(a[j], H, b[j]);
      }
    }
    ends[buf][stretch][lane] = make_float2(A, H);
    __syncthreads();                                 // (the other buffer's readers are past their loop: one barrier a round)
    float mine = S;
#pragma unroll 8
    for (int w = 0; w < n_stretches; w++) {
      if (w == stretch) mine = S;
      const float2 e = ends[buf][w][lane];
      S = fmaf(e.x, S, e.y);
    }
    T* po = (T*)P.out + (size_t)t0 * P.ldo + cc;
#pragma unroll
    for (int j = 0; j < LS_TOKENS; j++) {
      mine = fmaf(a[j], mine, b[j]);
      if (live && t0 + j < r1) po[(size_t)(j * P.ldo)] = from_float<T>(mine * lru_gelu<FAST>(yv[j]));
    }
  }
  if (P.write_state && live && stretch == 0) {
    slot[c] = S;
    const int keep = min(P.taps, r1 - r0);           // the ring takes the step's last inputs
    for (int k = 0; k < keep; k++) {
      const int t = r1 - 1 - k;
      slot[(size_t)(1 + P.token_pos[t] % P.taps) * P.width + c] = P.x[(size_t)t * P.ld + c];
    }
  }
}

// ---------------------------------------------------------------- decode steps: everything in one kernel
// A CTA of eight warps owns 32 channels of a block and up to 16 sequences.  It forms the block's u for its sequences in
// shared memory (every CTA of the block does: the ring makes that safe, see above), in two bfloat16 parts.  A warp then
// multiplies sixteen rows of the gates' matrices, eight channels' r and i, over one half of k: mma.sync.m16n8k16 with the
// weights as the A operand, so that a lane ends up with r and i of the same channel and sequences.  Weights are asked for
// before the kernel in front is waited for.
#define LT_WARPS 8
#define LT_CHANNELS 32
#define LT_SEQS 16
#define LT_AHEAD 4            // chunks of 32 values of k whose weights are in flight

__host__ __device__ __forceinline__ int lt_stride(int size) {    // bytes per row of u in shared memory: = 64 mod 128
  int s = ((size * 2 + 15) / 16) * 16;
  while (s % 128 != 64) s += 16;
  return s;
}

__global__ void __launch_bounds__(LT_WARPS * 32) lru_step_kernel(const Lru P) {
  extern __shared__ __align__(16) unsigned char lt_smem[];
  const int size = P.width / P.blocks;
  const int stride = lt_stride(size);
  unsigned char* u_hi = lt_smem;                                 // [LT_SEQS][stride]
  unsigned char* u_lo = u_hi + LT_SEQS * stride;
  float* u_own = reinterpret_cast<float*>(u_lo + LT_SEQS * stride);         // [LT_SEQS][LT_CHANNELS]
  float* part = u_own + LT_SEQS * LT_CHANNELS;                   // [4][2][4][32]: the second half of k's sums
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int quad = warp & 3, half = warp >> 2;
  const int b = blockIdx.y, c0 = blockIdx.x * LT_CHANNELS, m0 = blockIdx.z * LT_SEQS;
  const int ch = c0 + 8 * quad + g;                              // this lane's channel within the block
  const bool ch_ok = ch < size;
  pdl_trigger();
  const bf16* w_r = (const bf16*)P.gate_w + ((size_t)b * 2 * size + (ch_ok ? ch : 0)) * size;
  const bf16* w_i = w_r + (size_t)size * size;
  const int chunks = (size + 31) / 32, per = (chunks + 1) / 2;
  const int k_begin = half * per, k_end = min(chunks, k_begin + per);
  const uint4 zero4 = make_uint4(0, 0, 0, 0);
  uint4 wr[LT_AHEAD], wi[LT_AHEAD];
  auto load_weights = [&](int c) {
#pragma unroll
    for (int q = 0; q < LT_AHEAD; q++) {
      const int k = 32 * (c + q) + 8 * t;
      const bool ok = ch_ok && c + q < k_end && k < size;
      wr[q] = ok ? __ldg((const uint4*)(w_r + k)) : zero4;
      wi[q] = ok ? __ldg((const uint4*)(w_i + k)) : zero4;
    }
  };
  load_weights(k_begin);
  pdl_wait();                // the projection and the state are the work of kernels before this one: ld_fresh

  // u of the block's channels, four at a time (size is a multiple of 8)
  const int quads = size / 4;
  for (int i = threadIdx.x; i < LT_SEQS * quads; i += LT_WARPS * 32) {
    const int m = i / quads, c = 4 * (i - m * quads), row = m0 + m;
    const int at = b * size + c;
    float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
    const int seq = row < P.n_tokens ? P.token_seq[row] : -1;
    if (seq >= 0) {
      const int pos = P.token_pos[row];
      const float* ring = P.state + (size_t)P.seq_slot[seq] * P.state_stride + P.width + at;
      u = *reinterpret_cast<const float4*>(P.conv_b + at);
      for (int j = 0; j < P.taps; j++) {             // oldest input first: the order of lru_conv_kernel
        const int back = P.taps - 1 - j;
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (back == 0) x = ld_fresh((const float4*)(P.x + (size_t)row * P.ld + at));
        else if (pos - back >= 0) x = ld_fresh((const float4*)(ring + (size_t)((pos - back) % P.taps) * P.width));
        const float4 w = *reinterpret_cast<const float4*>(P.conv_w + (size_t)j * P.width + at);
        u.x = fmaf(w.x, x.x, u.x); u.y = fmaf(w.y, x.y, u.y); u.z = fmaf(w.z, x.z, u.z); u.w = fmaf(w.w, x.w, u.w);
      }
    }
    uint2 hi, lo;
    split_bf16(u, hi, lo);
    *reinterpret_cast<uint2*>(u_hi + (size_t)m * stride + 2 * c) = hi;
    *reinterpret_cast<uint2*>(u_lo + (size_t)m * stride + 2 * c) = lo;
    if (c >= c0 && c < c0 + LT_CHANNELS) *reinterpret_cast<float4*>(u_own + m * LT_CHANNELS + c - c0) = u;
  }
  __syncthreads();

  float acc[2][4];           // sequences 8 n + 2t, 2t + 1: r, r, i, i of channel ch
#pragma unroll
  for (int n = 0; n < 2; n++) { acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f; }
  for (int c = k_begin; c < k_end; c += LT_AHEAD) {
#pragma unroll
    for (int q = 0; q < LT_AHEAD; q++) {
      const int k = 32 * (c + q) + 8 * t;
      if (c + q >= k_end) break;
      const bool ok = k < size;
#pragma unroll
      for (int n = 0; n < 2; n++) {
        const size_t at = (size_t)(8 * n + g) * stride + 2 * k;
        const uint4 h = ok ? *reinterpret_cast<const uint4*>(u_hi + at) : zero4;
        const uint4 l = ok ? *reinterpret_cast<const uint4*>(u_lo + at) : zero4;
        mma16816(acc[n], wr[q].x, wi[q].x, wr[q].y, wi[q].y, h.x, h.y);
        mma16816(acc[n], wr[q].z, wi[q].z, wr[q].w, wi[q].w, h.z, h.w);
        mma16816(acc[n], wr[q].x, wi[q].x, wr[q].y, wi[q].y, l.x, l.y);
        mma16816(acc[n], wr[q].z, wi[q].z, wr[q].w, wi[q].w, l.z, l.w);
      }
    }
    if (c + LT_AHEAD < k_end) load_weights(c + LT_AHEAD);
  }
  if (half == 1) {
#pragma unroll
    for (int n = 0; n < 2; n++)
#pragma unroll
      for (int e = 0; e < 4; e++) part[((quad * 2 + n) * 4 + e) * 32 + lane] = acc[n][e];
  }
  __syncthreads();
  if (half == 1 || !ch_ok) return;
  const int chan = b * size + ch;
  const float rate = P.rate[chan], bias_r = P.gate_b[(size_t)b * 2 * size + ch], bias_i = P.gate_b[(size_t)b * 2 * size + size + ch];
#pragma unroll
  for (int n = 0; n < 2; n++)
#pragma unroll
    for (int e = 0; e < 2; e++) {
      const int m = 8 * n + 2 * t + e, row = m0 + m;
      if (row >= P.n_tokens) continue;
      const int seq = P.token_seq[row];
      bf16* o = (bf16*)P.out + (size_t)row * P.ldo + chan;
      if (seq < 0) { *o = __float2bfloat16_rn(0.f); continue; }
      const float rp = acc[n][e] + part[((quad * 2 + n) * 4 + e) * 32 + lane];
      const float ip = acc[n][2 + e] + part[((quad * 2 + n) * 4 + 2 + e) * 32 + lane];
      float* slot = P.state + (size_t)P.seq_slot[seq] * P.state_stride;
      const float2 ab = lru_coefficients<true>(rp + bias_r, ip + bias_i, u_own[m * LT_CHANNELS + ch - c0], rate);
      const float S = fmaf(ab.x, ld_fresh(slot + chan), ab.y);
      *o = __float2bfloat16_rn(S * lru_gelu<true>(ld_fresh(P.y + (size_t)row * P.ld + chan)));
      if (P.write_state) {
        slot[chan] = S;
        slot[(size_t)(1 + P.token_pos[row] % P.taps) * P.width + chan] = ld_fresh(P.x + (size_t)row * P.ld + chan);
      }
    }
}

static int lru_check(const Lru& P) {
  if (P.width < 1 || P.blocks < 1 || P.width % P.blocks != 0 || P.taps < 1) return STRATUM_ERR_SHAPE;
  if (P.ld < P.width || P.ldo < P.width) return STRATUM_ERR_SHAPE;
  if ((long long)P.state_stride < (1LL + P.taps) * P.width) return STRATUM_ERR_SHAPE;
  if (P.n_seqs > 65535 || P.blocks > 65535) return STRATUM_ERR_LIMIT;
  return 0;
}
static int lru_check_tensor_cores(const Lru& P) {
  if ((P.width / P.blocks) % 8 != 0 || P.ld % 4 != 0 || P.state_stride % 4 != 0) return STRATUM_ERR_SHAPE;
  const uintptr_t bits = (uintptr_t)P.y | (uintptr_t)P.x | (uintptr_t)P.gate_w | (uintptr_t)P.conv_w | (uintptr_t)P.conv_b |
                         (uintptr_t)P.state | (uintptr_t)P.u | (uintptr_t)P.pre;
  return (bits & 15) != 0 ? STRATUM_ERR_ALIGN : 0;
}

STRATUM_EXPORT int stratum_lru_conv(const Lru* params, cudaStream_t stream) {
  const Lru& P = *params;
  if (P.n_tokens <= 0) return 0;
  const int bad = lru_check(P);
  if (bad) return bad;
  const uintptr_t bits = (uintptr_t)P.x | (uintptr_t)P.u | (uintptr_t)P.conv_w | (uintptr_t)P.conv_b | (uintptr_t)P.state;
  if (P.width % 4 == 0 && P.ld % 4 == 0 && P.state_stride % 4 == 0 && (bits & 15) == 0 && P.taps >= 2 && P.taps <= 4) {
    const dim3 g4((P.n_tokens + LRU_RUN - 1) / LRU_RUN, (P.width / 4 + LRU_CONV_THREADS - 1) / LRU_CONV_THREADS);
    if (g4.y > 65535) return STRATUM_ERR_LIMIT;
    if (P.taps == 2) launch_pdl(lru_conv_vec_kernel<2>, g4, LRU_CONV_THREADS, 0, stream, P);
    else if (P.taps == 3) launch_pdl(lru_conv_vec_kernel<3>, g4, LRU_CONV_THREADS, 0, stream, P);
    else launch_pdl(lru_conv_vec_kernel<4>, g4, LRU_CONV_THREADS, 0, stream, P);
    return launch_status();
  }
  const dim3 grid((P.n_tokens + LRU_RUN - 1) / LRU_RUN, (P.width + LRU_CONV_THREADS - 1) / LRU_CONV_THREADS);
  if (grid.y > 65535) return STRATUM_ERR_LIMIT;
  switch (P.taps) {
    case 2: launch_pdl(lru_conv_kernel<2>, grid, LRU_CONV_THREADS, 0, stream, P); break;
    case 3: launch_pdl(lru_conv_kernel<3>, grid, LRU_CONV_THREADS, 0, stream, P); break;
    case 4: launch_pdl(lru_conv_kernel<4>, grid, LRU_CONV_THREADS, 0, stream, P); break;
    default: launch_pdl(lru_conv_kernel<0>, grid, LRU_CONV_THREADS, 0, stream, P); break;
  }
  return launch_status();
}

// The gates' pre-activations of every token from u, bfloat16 matrices.  Needs width / blocks % 8 == 0.
STRATUM_EXPORT int stratum_lru_gates(const Lru* params, cudaStream_t stream) {
  const Lru& P = *params;
  if (P.n_tokens <= 0) return 0;
  int bad = lru_check(P);
  if (!bad) bad = lru_check_tensor_cores(P);
  if (bad) return bad;
  const int two = 2 * (P.width / P.blocks);
  const dim3 grid((P.n_tokens + LG_M - 1) / LG_M, (two + LG_N - 1) / LG_N, P.blocks);
  if (grid.y > 65535) return STRATUM_ERR_LIMIT;
  const size_t smem = 2 * LG_STAGE * sizeof(bf16);
  cudaError_t e = cudaFuncSetAttribute(lru_gates_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  launch_pdl(lru_gates_kernel, grid, 256, smem, stream, P);
  return launch_status();
}

STRATUM_EXPORT int stratum_lru_scan(const Lru* params, int out_dtype, cudaStream_t stream) {
  const Lru& P = *params;
  if (P.n_tokens <= 0 || P.n_seqs <= 0) return 0;
  const int bad = lru_check(P);
  if (bad) return bad;
  int warps = (P.max_new + 2 * LS_TOKENS - 1) / (2 * LS_TOKENS);
  warps = warps < 1 ? 1 : (warps > LS_MAX_WARPS ? LS_MAX_WARPS : warps);
  const dim3 grid((P.width + LS_CHANNELS - 1) / LS_CHANNELS, P.n_seqs);
  if (out_dtype == STRATUM_DT_F32) lru_scan_kernel<float><<<grid, warps * 32, 0, stream>>>(P);
  else if (out_dtype == STRATUM_DT_BF16) lru_scan_kernel<bf16><<<grid, warps * 32, 0, stream>>>(P);
  else return STRATUM_ERR_DTYPE;
  return launch_status();
}

// A step that brings one token per sequence, bfloat16 out and matrices.  Needs width / blocks % 8 == 0.
STRATUM_EXPORT int stratum_lru_step(const Lru* params, cudaStream_t stream) {
  const Lru& P = *params;
  if (P.n_tokens <= 0) return 0;
  int bad = lru_check(P);
  if (!bad) bad = lru_check_tensor_cores(P);
  if (bad) return bad;
  const int size = P.width / P.blocks;
  const size_t smem = 2LL * LT_SEQS * lt_stride(size) + (LT_SEQS * LT_CHANNELS + 4 * 2 * 4 * 32) * sizeof(float);
  if (smem > 200 * 1024) return STRATUM_ERR_LIMIT;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(lru_step_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  const dim3 grid((size + LT_CHANNELS - 1) / LT_CHANNELS, P.blocks, (P.n_tokens + LT_SEQS - 1) / LT_SEQS);
  if (grid.z > 65535) return STRATUM_ERR_LIMIT;
  launch_pdl(lru_step_kernel, grid, LT_WARPS * 32, smem, stream, P);
  return launch_status();
}
