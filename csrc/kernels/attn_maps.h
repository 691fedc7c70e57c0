// Arguments shared by the kernels of attention with several score maps over one set of values (differential
// attention): query head h and key head g hold `maps` vectors of `dim` each, laid out [map 0, map 1] and padded to
// dim_p; every map has its own scores and softmax over the value head's `vdim` columns (padded to vdim_p).  With two
// maps the head's result is
//     o = a_0 - lambda * a_1;     o <- out_scale * o / sqrt(mean(o^2) + eps)
// and with one map it is a_0.  softcap > 0 replaces a score s by softcap * tanh(s / softcap); window > 0 limits a query to
// itself and the window - 1 tokens before it.
#pragma once

struct NkbMapsArgs {
  int maps, heads, kv_heads, dim, dim_p, vdim, vdim_p;
  float scale, softcap, lambda, out_scale, eps;
  int window;
};
