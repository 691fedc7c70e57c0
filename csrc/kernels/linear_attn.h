// Arguments of the linear-attention kernels (linear_attn.cu): heads with a [dim x vdim] state that decays per key channel,
//
//   read after the update     S_t = diag(a_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T (q_scale q_t)            (bonus == nullptr)
//   read before the update    o_t = (S_(t-1) + diag(bonus) k_t v_t^T)^T (q_scale q_t),   then S_t as above
//
// with the decay of channel c from a logit z[c] = z_bias[c] + (w2 z_act(x))[c], x the low-rank input (or z itself when w2 is
// null), and each head's result o turned into
//
//   out_scale * gate_act(g) * norm_w * o / sqrt(mean(o^2) + eps).
#pragma once
#include "proj_src.h"

enum { NKB_DECAY_SIGMOID = 0 /* sigmoid(z)^inv_tau */, NKB_DECAY_DOUBLE_EXP = 1 /* exp(-exp(z)) */ };

struct NkbLinAttn {
  NkbProj q, k, v, z, g;
  const void* w2;           // [heads * dim, rank] or nullptr
  const float* z_bias;      // [heads * dim]
  const float* bonus;       // [heads * dim] or nullptr
  const float* norm_w;      // element h * norm_stride + j
  float* state;             // [slots, heads, vdim, dim_p], dim_p = dim rounded up to a multiple of 4
  const int* slot_ids;      // [batch] or nullptr (slot = batch index)
  const int* q_start;       // scan only
  const int* q_lens;        // scan only
  const int* context_lens;  // counts the new tokens; negative = inactive
  void* heads_out;          // scan only: [tokens, heads * vdim], room for the heads before norm and gate
  void* out;                // [tokens, out_ld]
  long long out_ld;
  int w2_bf16, rank, z_act, decay, norm_stride, gate_act, bf16;
  int batch, tokens, heads, dim, vdim;
  float q_scale, inv_tau, out_scale, eps;
};
