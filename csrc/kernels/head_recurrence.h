// Arguments of the recurrences whose [dim x vdim] state decays by one number per head (head_recurrence.cu), fed through a short
// causal convolution per channel.  With g_t = exp(-rate * softplus(a_t + dt_bias)), per head
//
//   delta rule (b set)       S <- g S;   u = sigmoid(b) (v - S^T k);    S <- S + k u^T;   o = S^T q
//                            (k divided by sqrt(sum k^2 + unit_eps), q likewise and multiplied by q_scale)
//   state space (b null)     S <- g S + k (softplus(a + dt_bias) v)^T;   o = S^T (q_scale q) + skip v
//
// Query / key head of head h: h / (heads / groups).  q, k and v are columns of one row of `channels` convolved channels:
// y_t[c] = silu(conv_b[c] + sum_j conv_w[j][c] x_(t - (taps - 1) + j)[c]).  The inputs of a sequence's last tokens stay in its
// slot, that of position p in row p % taps: a decode step writes a row that nobody reads in it.
#pragma once
#include "proj_src.h"

struct NkbHeadRec {
  NkbProj x;                // step: channels before the convolution; scan: after it (finished values)
  NkbProj a, b;             // [tokens, heads]; b.ptr null: state space form
  NkbProj g;                // step with norm_w: output gates [tokens, heads * vdim]
  const float* conv_w;      // [taps, channels]
  const float* conv_b;      // [channels] or null
  float* conv_state;        // [slots, taps, channels]
  const float* rate;        // [heads]
  const float* dt_bias;     // [heads]
  const float* skip;        // [heads] or null
  const float* norm_w;      // [vdim]: the step finishes its heads, gate_act(g) * norm_w * o / sqrt(mean(o^2) + eps); or null
  float* state;             // [slots, heads, vdim, dim_p], dim_p = dim rounded up to a multiple of 4
  const int* slot_ids;      // [batch] or null (slot = batch index)
  const int* q_start;       // scan only
  const int* q_lens;        // scan only
  const int* context_lens;  // counts the new tokens; negative = inactive
  void* out;                // [tokens, heads * vdim]; without norm_w the step writes fp32
  int taps, channels, q_col, k_col, v_col, gate_act, bf16;
  int batch, tokens, heads, groups, dim, vdim;
  float q_scale, eps, unit_eps;
};
