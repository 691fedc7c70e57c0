// Where a kernel finds one slice of a projection's result.  The layers of a mixed decoder hand their
// projections on in three forms: fp32 split-K partial sums [splits][tokens][ld] (decode-sized batches), a
// bf16 matrix [tokens][ld] (prefill-sized ones) or an fp32 matrix (32-bit models, the same as one split).
// `ptr` already points at the slice's first column.
#pragma once

struct NkbProj {
  const void* ptr;
  long long ld;             // elements between two tokens
  long long split_stride;   // elements between two partial sums (fp32 only)
  int splits;               // 1 for finished values
  int bf16;                 // 1 = bf16 values, 0 = fp32
};

// One addend of a residual update: scale * y, with a gate sigmoid(g + gbias) on it when g.ptr is set (token_gate: one g per
// token, no bias), or (pair_pos set) the sum of a token's top_k rows of y, pair_w[t, j] * y[pair_pos[t, j]] (routed experts;
// pair_w null: weights of one), or (norm_w set) norm_w * y / sqrt(mean(y^2) + eps).
struct NkbBranch {
  NkbProj y, g;
  const float* gbias;
  const int* pair_pos;
  const float* pair_w;
  const float* norm_w;
  int top_k, token_gate;
  float scale;
};
