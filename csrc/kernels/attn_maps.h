// Arguments shared by the kernels of attention with several score maps over one set of values (differential
// attention): query head h and key head g hold `maps` vectors of `dim` each, laid out [map 0, map 1] and padded to
// dim_p; every map has its own scores and softmax over the value head's `vdim` columns (padded to vdim_p).  With two
// maps the head's result is
//     o = a_0 - lambda * a_1;     o <- out_scale * o / sqrt(mean(o^2) + eps)
// and with one map it is a_0.  softcap > 0 replaces a score s by softcap * tanh(s / softcap); window > 0 limits a query to
// itself and the window - 1 tokens before it (and the first keep_first tokens), chunk > 0 to the tokens of its own chunk of that
// many positions; sinks holds per head (one map) the logarithm of an addend of the softmax's denominator.  dist_a and dist_b, per
// head (one map): after the cap a score loses dist_a * ln(1 + dist_b * distance).
#pragma once

struct NkbMapsArgs {
  int maps, heads, kv_heads, dim, dim_p, vdim, vdim_p;
  float scale, softcap, lambda, out_scale, eps;
  int window, chunk;
  const float* sinks;                    // [heads] or null
  // elements between tokens / heads of queries and results, 0: one token's heads side by side
  long long q_token, q_head, o_token, o_head;
  int v_ld;                              // elements between the values of two tokens, 0: vdim_p (values inside wider rows)
  int keep_first;                        // with a window: the first tokens every query sees
  const float *dist_a, *dist_b;          // [heads] or null
};

// What the kernels of plain attention (attn_prefill.cu, attn_decode.cu) do to a score beyond scaling it.
struct NkbScoreMods {
  float softcap;                         // <= 0: none
  int keep_first;
  const float *dist_a, *dist_b;
};

// First position a query at `pos` sees (kept first tokens aside).
static inline
#ifdef __CUDACC__
__host__ __device__
#endif
int nkb_first_visible(int pos, int window, int chunk) {
  int lo = window > 0 && pos >= window ? pos - window + 1 : 0;
  if (chunk > 0 && pos - pos % chunk > lo) lo = pos - pos % chunk;
  return lo;
}
