// Arguments shared by the kernels of latent attention: all heads read one row per token, the latent c of `rank` elements and a
// rotated key part of `rot` elements behind it, padded to `row` elements in the cache.  A query head is `dim` unrotated and
// `rot` rotated elements.  Per head h the key is [W_uk[h] c, rotated part] and the value W_uv[h] c; with the query folded
// through W_uk[h] the scores are products with the cached row itself and the result is a mixture of latents.
#pragma once

struct NkbLatentArgs {
  int heads, dim, rot, rank, q_rank, row;
  float eps, scale;
  int window;                            // > 0: a query sees itself and the window - 1 tokens before it
  const float* sinks;                    // [heads] or null: logarithms of an addend of the softmax's denominator
  // elements between two tokens and two heads of the queries [.., row] and of the results [.., rank]
  long long q_token, q_head, o_token, o_head;
};
