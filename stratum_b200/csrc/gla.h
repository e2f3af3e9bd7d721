// What the kernels of gated linear attention, retention and lightning attention are told (mirrored field by field by kernels.py: pointers
// first, then 4-byte fields).  See gla.cu for the meaning of every field.
#pragma once
#include "common.cuh"

#define GLA_ROWS 16           // rows of a column of S that a lane of the recurrence holds

struct Gla {
  const float* proj;        // [tokens][ld]
  void* inner;              // [tokens][ld_inner], the compute dtype: the decay's inner projection (cast)
  const float* head_decay;  // [n_heads] or null: the decays are alpha's
  const float* gain;        // [vdim] ([n_heads * vdim] with norm_all), or null: none
  float* alpha;             // [tokens][n_heads * dim]: z when `decay` begins, alpha when it ends
  float* o_raw;             // [tokens][n_heads * vdim]
  void* out;                // [tokens][ldo] compute dtype
  float* state;             // [slots][state_stride]: S^T [n_heads][vdim][dim]
  const int* token_seq;
  const int* seq_start;     // [seqs + 1]
  const int* seq_slot;      // [seqs]
  int ld, ldo, n_tokens, n_seqs;
  int n_heads, dim, vdim, rank;
  int state_stride, write_state, ld_inner, rot_pairs;
  float eps, inv_tau, q_scale;
  int silu_qkv;             // q, k and v are taken through silu when they are read
  int norm_all;             // finish: one norm over all heads together, gated by sigmoid(g) (0: a norm per head, silu(g))
};

static int gla_check(const Gla& P) {
  if (P.n_heads < 1 || P.dim < 1 || P.vdim < 1 || P.rank < (P.head_decay ? 0 : 1)) return STRATUM_ERR_SHAPE;
  if (P.ld < 2 * P.n_heads * P.dim + 2 * P.n_heads * P.vdim + P.rank || P.ldo < P.n_heads * P.vdim)
    return STRATUM_ERR_SHAPE;
  if (P.state_stride < P.n_heads * P.dim * P.vdim) return STRATUM_ERR_SHAPE;
  if (P.dim > 32 * GLA_ROWS) return STRATUM_ERR_LIMIT;
  if (P.n_heads > 65535 || P.n_seqs > 65535) return STRATUM_ERR_LIMIT;
  return 0;
}
