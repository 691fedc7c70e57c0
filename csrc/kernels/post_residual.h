// Arguments of the residual update whose branches pass a norm before they are added (post_residual.cu):
//
//   s      = sum over branches of scale * (y + shift), or with norm_w scale * norm_w * (y + shift) / sqrt(mean((y + shift)^2) + eps)
//   r      = x (or table[id] * table_scale) + post(s)
//   x_out  = sum over j < past of coef[j] * history[j], + coef[past] * r          (coef null: r)
//   out_n  = norm_n(x_out)
//
// A norm here is the elementwise tanh(alpha x) * w + b; w null: x itself.
#pragma once
#include "proj_src.h"

struct NkbTanhNorm {
  const float* w;
  const float* b;
  float alpha;
  void* out;                // norms of the sum only
};

struct NkbPostBranch {
  NkbProj y;
  const float* shift;       // [width] or null
  const float* norm_w;      // [width] or null
  float scale;
};

struct NkbPostResidual {
  const float* x_in;        // fp32 rows, or null with ids / table
  const int* ids;
  const void* table;        // [vocab, width], bf16 or fp32
  NkbPostBranch br[2];
  NkbTanhNorm post, norm[2];
  const float* history;     // [past] matrices, history_stride elements apart
  const float* coef;        // [past + 1] or null
  float* result;            // r, or null
  float* x_out;             // or null
  long long history_stride;
  int vocab, table_bf16, branches, norms, past, out_bf16, rows, width;
  float table_scale, eps;
};
