// Attention with several score maps over shared values (attn_maps.h), everything but the tensor-core prefill:
//   append   interleaved partial rotary embedding of queries and keys from the fused projection, keys and values
//            into their slots of the paged cache
//   row norm append   the same for one map without rotation, queries and keys normed over all heads of the token together
//   rope norm append   the same for one map with projection biases, rotated or not (pairs half a rotated part apart, or next to
//            each other), with or without an RMS norm without weight over every head of queries and keys; without keys for
//            layers that read another layer's
//   decode   one new token per sequence, bf16: the two maps of up to eight query heads are the sixteen rows of
//            one MMA fragment (rows 0-7 map 0, rows 8-15 map 1).  A key row holds both maps' keys side by side, so with
//            the query of map 0 only in the first half of the contraction and that of map 1 only in the second, one
//            accumulator receives both maps' scores, and both maps share every value fragment.  TMA page ring,
//            splits and their merge as in attn_decode.cu; the maps are combined and normalised after the merge.
//   simple   any sizes, any storage type, any number of new tokens: one CTA per (token, head), scores and softmax
//            on the CUDA cores in fp32.  Serves 32-bit models and head sizes the tiled kernels do not take.
// Cache: keys [block, kv_head, 32, maps * dim_p], values [block, kv_head, 32, vdim_p]; padding columns are zero.
#include "common.cuh"
#include "mma_frag.cuh"
#include "proj_src.cuh"
#include "attn_maps.h"
#include "api.h"
#include <math.h>

namespace nkb {

constexpr int kMapsPage = 32;

// ------------------------------------------------------------------------------------------------ append
struct MapsAppendParams {
  NkbProj q, k, v;
  NkbMapsArgs a;
  const float* cos_sin;     // [max_pos, rot_dims]: cos of the rot_dims / 2 angles, then sin (scaling included)
  const int* positions;
  const int* slots;
  void *q_out, *k_cache, *v_cache;
  int rot_dims, max_pos, tokens;
  int vec;                  // sizes and alignments allow four elements at a time
};

template <typename T>
__device__ __forceinline__ void store4(T* dst, float4 x) {
  if constexpr (sizeof(T) == 2)
    *reinterpret_cast<uint2*>(dst) = make_uint2(pack_bf16x2(x.x, x.y), pack_bf16x2(x.z, x.w));
  else
    *reinterpret_cast<float4*>(dst) = x;
}

template <typename T>
__global__ void __launch_bounds__(256) maps_append_kernel(const __grid_constant__ MapsAppendParams p) {
  const int units = p.a.heads + 2 * p.a.kv_heads;
  const long long gw = (blockIdx.x * 256ll + threadIdx.x) >> 5;
  const int lane = threadIdx.x & 31;
  griddep_wait();
  griddep_launch();
  if (gw >= (long long)p.tokens * units) return;
  const int t = int(unsigned(gw) / unsigned(units)), u = int(unsigned(gw) % unsigned(units));
  const bool is_q = u < p.a.heads, is_v = u >= p.a.heads + p.a.kv_heads;
  const int slot = p.slots[t];
  if (!is_q && slot < 0) return;
  const long long blk = slot / kMapsPage, off = slot % kMapsPage;
  if (is_v) {
    const int h = u - p.a.heads - p.a.kv_heads;
    T* dst = reinterpret_cast<T*>(p.v_cache) + ((blk * p.a.kv_heads + h) * kMapsPage + off) * p.a.vdim_p;
    if (p.vec) {
      for (int c = lane * 4; c < p.a.vdim; c += 128) store4<T>(dst + c, proj_load4(p.v, t, h * p.a.vdim + c));
      return;
    }
    for (int c = lane; c < p.a.vdim; c += 32) dst[c] = cast_out<T>(proj_load(p.v, t, h * p.a.vdim + c));
    return;
  }
  const int h = is_q ? u : u - p.a.heads;
  const int kw = p.a.maps * p.a.dim_p;
  T* dst = is_q ? reinterpret_cast<T*>(p.q_out) + ((long long)t * p.a.heads + h) * kw
                : reinterpret_cast<T*>(p.k_cache) + ((blk * p.a.kv_heads + h) * kMapsPage + off) * kw;
  const NkbProj& src = is_q ? p.q : p.k;
  const int pos = min(max(p.positions[t], 0), p.max_pos - 1);
  const float* cs = p.cos_sin + (long long)pos * p.rot_dims;
  const int quarter = p.a.dim_p / 4;
  if (p.vec) {
    // four consecutive elements (two pairs) per lane
    for (int i = lane; i < p.a.maps * quarter; i += 32) {
      const int m = i / quarter, c = (i % quarter) * 4;
      float4 x = c < p.a.dim ? proj_load4(src, t, (h * p.a.maps + m) * p.a.dim + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < p.rot_dims) {
        const float2 co = *reinterpret_cast<const float2*>(cs + (c >> 1));
        const float2 si = *reinterpret_cast<const float2*>(cs + (p.rot_dims >> 1) + (c >> 1));
        x = make_float4(x.x * co.x - x.y * si.x, x.y * co.x + x.x * si.x, x.z * co.y - x.w * si.y, x.w * co.y + x.z * si.y);
      }
      store4<T>(dst + m * p.a.dim_p + c, x);
    }
    return;
  }
  const int half = p.a.dim_p / 2;
  for (int i = lane; i < p.a.maps * half; i += 32) {
    const int m = i / half, c = (i % half) * 2;         // pair (c, c + 1) of map m
    const int col = (h * p.a.maps + m) * p.a.dim + c;
    float x = c < p.a.dim ? proj_load(src, t, col) : 0.f;
    float y = c + 1 < p.a.dim ? proj_load(src, t, col + 1) : 0.f;
    if (c < p.rot_dims) {
      const float co = cs[c >> 1], si = cs[(p.rot_dims >> 1) + (c >> 1)];
      const float r = x * co - y * si;
      y = y * co + x * si;
      x = r;
    }
    dst[m * p.a.dim_p + c] = cast_out<T>(x);
    dst[m * p.a.dim_p + c + 1] = cast_out<T>(y);
  }
}

// One CTA per token: RMS norms over the whole query and the whole key projection (weights of their full widths), queries
// out with zeroed padding, keys and values into the cache.
struct RowNormAppendParams {
  NkbProj q, k, v;
  NkbMapsArgs a;
  const float *q_norm, *k_norm;
  const int* slots;
  void *q_out, *k_cache, *v_cache;
};

template <int V, typename T>
__device__ __forceinline__ void store_v(T* dst, const float (&x)[V]) {
  if constexpr (V == 4) {
    store4<T>(dst, make_float4(x[0], x[1], x[2], x[3]));
  } else {
    *dst = cast_out<T>(x[0]);
  }
}
template <int V>
__device__ __forceinline__ void load_v(float (&x)[V], const NkbProj& s, long long row, int c) {
  if constexpr (V == 4) {
    const float4 r = proj_load4(s, row, c);
    x[0] = r.x; x[1] = r.y; x[2] = r.z; x[3] = r.w;
  } else {
    x[0] = proj_load(s, row, c);
  }
}

template <int V, typename T>
__global__ void __launch_bounds__(256) row_norm_append_kernel(const __grid_constant__ RowNormAppendParams p) {
  extern __shared__ __align__(16) float rn_s[];   // q row, k row
  __shared__ float red[2][8];
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int nq = p.a.heads * p.a.dim, nk = p.a.kv_heads * p.a.dim, nv = p.a.kv_heads * p.a.vdim;
  griddep_wait();
  griddep_launch();
  const int slot = p.slots[t];
  const long long blk = slot < 0 ? 0 : slot / kMapsPage, off = slot < 0 ? 0 : slot % kMapsPage;
  float sq = 0.f, sk = 0.f;
  for (int c = threadIdx.x * V; c < nq; c += 256 * V) {
    float x[V];
    load_v<V>(x, p.q, t, c);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      sq += x[j] * x[j];
      rn_s[c + j] = x[j];
    }
  }
  for (int c = threadIdx.x * V; c < nk; c += 256 * V) {
    float x[V];
    load_v<V>(x, p.k, t, c);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      sk += x[j] * x[j];
      rn_s[nq + c + j] = x[j];
    }
  }
  if (slot >= 0) {
    T* vc = reinterpret_cast<T*>(p.v_cache);
    for (int c = threadIdx.x * V; c < nv; c += 256 * V) {
      float x[V];
      load_v<V>(x, p.v, t, c);
      const int h = c / p.a.vdim, d = c % p.a.vdim;
      store_v<V, T>(vc + ((blk * p.a.kv_heads + h) * kMapsPage + off) * p.a.vdim_p + d, x);
    }
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if (lane == 0) {
    red[0][warp] = sq;
    red[1][warp] = sk;
  }
  __syncthreads();
  float tq = 0.f, tk = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) {
    tq += red[0][w];
    tk += red[1][w];
  }
  const float iq = 1.f / sqrtf(tq / float(nq) + p.a.eps), ik = 1.f / sqrtf(tk / float(nk) + p.a.eps);
  T* qo = reinterpret_cast<T*>(p.q_out) + (long long)t * p.a.heads * p.a.dim_p;
  for (int i = threadIdx.x * V; i < p.a.heads * p.a.dim_p; i += 256 * V) {
    const int h = i / p.a.dim_p, d = i % p.a.dim_p;
    float x[V];
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const int c = h * p.a.dim + d + j;
      x[j] = d + j < p.a.dim ? rn_s[c] * iq * p.q_norm[c] : 0.f;
    }
    store_v<V, T>(qo + i, x);
  }
  if (slot < 0) return;
  T* kc = reinterpret_cast<T*>(p.k_cache);
  for (int c = threadIdx.x * V; c < nk; c += 256 * V) {
    const int h = c / p.a.dim, d = c % p.a.dim;
    float x[V];
#pragma unroll
    for (int j = 0; j < V; ++j) x[j] = rn_s[nq + c + j] * ik * p.k_norm[c + j];
    store_v<V, T>(kc + ((blk * p.a.kv_heads + h) * kMapsPage + off) * p.a.dim_p + d, x);
  }
}

// One warp per (token, head of queries / keys / values).
struct RopeNormAppendParams {
  NkbProj q, k, v;          // k.ptr null: queries only
  NkbMapsArgs a;
  const float* bias;        // [heads * dim (+ kv_heads * dim + kv_heads * vdim)] or null
  const float* cos_sin;     // [max_pos, rot_dims]: cos of the rot_dims / 2 angles, then sin
  const int *positions, *slots;
  void *q_out, *k_cache, *v_cache;
  int rot_dims, max_pos, tokens, norm;
  int pairs;                // rotation of pairs (2i, 2i + 1) instead of (i, i + rot_dims / 2)
};

template <int V>
__device__ __forceinline__ void add_bias(float (&x)[V], const float* bias, int c) {
  if (!bias) return;
#pragma unroll
  for (int j = 0; j < V; ++j) x[j] += bias[c + j];
}

template <int V, typename T>
__global__ void __launch_bounds__(256) rope_norm_append_kernel(const __grid_constant__ RopeNormAppendParams p) {
  const int units = p.a.heads + (p.k.ptr ? 2 * p.a.kv_heads : 0), dim = p.a.dim;
  const long long gw = (blockIdx.x * 256ll + threadIdx.x) >> 5;
  const int lane = threadIdx.x & 31;
  griddep_wait();
  griddep_launch();
  if (gw >= (long long)p.tokens * units) return;
  const int t = int(unsigned(gw) / unsigned(units)), u = int(unsigned(gw) % unsigned(units));
  const bool is_q = u < p.a.heads, is_v = u >= p.a.heads + p.a.kv_heads;
  const int slot = is_q ? 0 : p.slots[t];
  if (slot < 0) return;
  const long long blk = slot / kMapsPage, off = slot % kMapsPage;
  if (is_v) {
    const int h = u - p.a.heads - p.a.kv_heads;
    const float* bias = p.bias ? p.bias + (p.a.heads + p.a.kv_heads) * dim + h * p.a.vdim : nullptr;
    T* dst = reinterpret_cast<T*>(p.v_cache) + ((blk * p.a.kv_heads + h) * kMapsPage + off) * p.a.vdim_p;
    for (int c = lane * V; c < p.a.vdim; c += 32 * V) {
      float x[V];
      load_v<V>(x, p.v, t, h * p.a.vdim + c);
      add_bias<V>(x, bias, c);
      store_v<V, T>(dst + c, x);
    }
    return;
  }
  const int h = is_q ? u : u - p.a.heads;
  const NkbProj& src = is_q ? p.q : p.k;
  const float* bias = p.bias ? p.bias + u * dim : nullptr;
  T* dst = is_q ? reinterpret_cast<T*>(p.q_out) + ((long long)t * p.a.heads + h) * p.a.dim_p
                : reinterpret_cast<T*>(p.k_cache) + ((blk * p.a.kv_heads + h) * kMapsPage + off) * p.a.dim_p;
  const int pos = min(max(p.positions[t], 0), p.max_pos - 1), n = p.rot_dims / 2;
  const float* cs = p.cos_sin + (long long)pos * p.rot_dims;
  const auto load = [&](float (&x)[V], int c) {
    load_v<V>(x, src, t, h * dim + c);
    add_bias<V>(x, bias, c);
  };
  const auto finish = [&](float (&x)[V], const float (&y)[V], int c, float inv) {       // y: the elements x is paired with
    if (p.pairs) {
      if (c < 2 * n) {
        if constexpr (V == 4) {
          const float2 co = *reinterpret_cast<const float2*>(cs + (c >> 1)), si = *reinterpret_cast<const float2*>(cs + n + (c >> 1));
          const float r0 = x[0] * co.x - x[1] * si.x, r2 = x[2] * co.y - x[3] * si.y;
          x[1] = x[1] * co.x + x[0] * si.x;
          x[3] = x[3] * co.y + x[2] * si.y;
          x[0] = r0;
          x[2] = r2;
        } else {
          x[0] = x[0] * cs[c >> 1] + ((c & 1) ? y[0] : -y[0]) * cs[n + (c >> 1)];
        }
      }
    } else if (c < 2 * n) {
      const int i = c < n ? c : c - n;
      const float sign = c < n ? -1.f : 1.f;
#pragma unroll
      for (int j = 0; j < V; ++j) x[j] = x[j] * cs[i + j] + sign * y[j] * cs[n + i + j];
    }
#pragma unroll
    for (int j = 0; j < V; ++j) x[j] *= inv;
    store_v<V, T>(dst + c, x);
  };
  // the rotation keeps a head's length, so the norm's sum is taken before it
  float x[V], ss = 0.f;
  if (dim <= 32 * V) {
    // a lane holds its elements; those it is paired with lie n / V lanes away
    const int c = lane * V;
#pragma unroll
    for (int j = 0; j < V; ++j) x[j] = 0.f;
    if (c < dim) load(x, c);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += x[j] * x[j];
    const float inv = p.norm ? 1.f / sqrtf(warp_sum(ss) / float(dim) + p.a.eps) : 1.f;
    const int from = p.pairs ? (V == 1 ? lane ^ 1 : lane) : c < n ? lane + n / V : (c < 2 * n ? lane - n / V : lane);
    float y[V];
#pragma unroll
    for (int j = 0; j < V; ++j) y[j] = __shfl_sync(0xffffffffu, x[j], from);
    if (c < p.a.dim_p) finish(x, y, c, inv);
    const float zero[V] = {};
    for (int z = c + 32 * V; z < p.a.dim_p; z += 32 * V) store_v<V, T>(dst + z, zero);
    return;
  }
  for (int c = lane * V; c < dim; c += 32 * V) {
    load(x, c);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += x[j] * x[j];
  }
  const float inv = p.norm ? 1.f / sqrtf(warp_sum(ss) / float(dim) + p.a.eps) : 1.f;
  for (int c = lane * V; c < p.a.dim_p; c += 32 * V) {
    float y[V];
#pragma unroll
    for (int j = 0; j < V; ++j) x[j] = y[j] = 0.f;
    if (c < dim) load(x, c);
    if (c < 2 * n) load(y, p.pairs ? (V == 1 ? c ^ 1 : c) : c < n ? c + n : c - n);
    finish(x, y, c, inv);
  }
}

// Prompts in bf16, sizes of whole 16-byte pieces, heads of at most 8 L elements: L lanes share a head of queries, keys or
// values, a lane holds eight elements of kRopeUnits heads and loads all of them first.
constexpr int kRopeUnits = 4;

template <int L>
__global__ void __launch_bounds__(256) rope_norm_append8_kernel(const __grid_constant__ RopeNormAppendParams p) {
  using bf = __nv_bfloat16;
  const int units = p.a.heads + (p.k.ptr ? 2 * p.a.kv_heads : 0), dim = p.a.dim, n = p.rot_dims / 2;
  const int lane = threadIdx.x & (L - 1), c = lane * 8, groups = 256 / L;
  griddep_wait();
  griddep_launch();
  const long long total = (long long)p.tokens * units, first = blockIdx.x * (long long)(groups * kRopeUnits) + threadIdx.x / L;
  uint4 raw[kRopeUnits];
  int tok[kRopeUnits], unit[kRopeUnits];
#pragma unroll
  for (int i = 0; i < kRopeUnits; ++i) {
    const long long w = first + i * groups;
    tok[i] = w < total ? int(unsigned(w) / unsigned(units)) : -1;
    unit[i] = w < total ? int(unsigned(w) % unsigned(units)) : 0;
    raw[i] = make_uint4(0u, 0u, 0u, 0u);
    if (tok[i] < 0) continue;
    const int u = unit[i];
    const bool is_v = u >= p.a.heads + p.a.kv_heads;
    const NkbProj& src = u < p.a.heads ? p.q : is_v ? p.v : p.k;
    const int h = u < p.a.heads ? u : is_v ? u - p.a.heads - p.a.kv_heads : u - p.a.heads;
    const int width = is_v ? p.a.vdim : dim;
    if (c < width) raw[i] = *reinterpret_cast<const uint4*>(reinterpret_cast<const bf*>(src.ptr) + tok[i] * src.ld + h * width + c);
  }
#pragma unroll
  for (int i = 0; i < kRopeUnits; ++i) {
    const int u = unit[i];
    const bool live = tok[i] >= 0, is_q = u < p.a.heads, is_v = u >= p.a.heads + p.a.kv_heads;
    const int slot = live && !is_q ? p.slots[tok[i]] : 0, width = is_v ? p.a.vdim : dim;
    float x[8];
    const uint32_t rw[4] = {raw[i].x, raw[i].y, raw[i].z, raw[i].w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 f = unpack_bf16x2(rw[e]);
      x[2 * e] = f.x;
      x[2 * e + 1] = f.y;
    }
    if (p.bias && live && c < width) {
      const float* b = p.bias + (is_v ? (p.a.heads + p.a.kv_heads) * dim + (u - p.a.heads - p.a.kv_heads) * p.a.vdim : u * dim) + c;
      const float4 lo = *reinterpret_cast<const float4*>(b), hi = *reinterpret_cast<const float4*>(b + 4);
      x[0] += lo.x; x[1] += lo.y; x[2] += lo.z; x[3] += lo.w;
      x[4] += hi.x; x[5] += hi.y; x[6] += hi.z; x[7] += hi.w;
    }
    float ss = 0.f, y[8];
    const int from = p.pairs ? lane : c < n ? lane + n / 8 : (c < 2 * n ? lane - n / 8 : lane);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      ss += x[e] * x[e];
      y[e] = __shfl_sync(0xffffffffu, x[e], from, L);
    }
#pragma unroll
    for (int w = L / 2; w > 0; w >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, w);
    if (!live || slot < 0) continue;
    const long long blk = slot / kMapsPage, off = slot % kMapsPage;
    bf* dst;
    int pad = p.a.dim_p;
    if (is_v) {
      dst = reinterpret_cast<bf*>(p.v_cache) + ((blk * p.a.kv_heads + u - p.a.heads - p.a.kv_heads) * kMapsPage + off) * p.a.vdim_p;
      pad = p.a.vdim;
    } else {
      const float inv = p.norm ? 1.f / sqrtf(ss / float(dim) + p.a.eps) : 1.f;
      if (p.pairs && c < 2 * n) {
        const float* cs = p.cos_sin + (long long)min(max(p.positions[tok[i]], 0), p.max_pos - 1) * p.rot_dims + (c >> 1);
        const float4 co = *reinterpret_cast<const float4*>(cs), si = *reinterpret_cast<const float4*>(cs + n);
        const float cv[4] = {co.x, co.y, co.z, co.w}, sv[4] = {si.x, si.y, si.z, si.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float r = x[2 * e] * cv[e] - x[2 * e + 1] * sv[e];
          x[2 * e + 1] = x[2 * e + 1] * cv[e] + x[2 * e] * sv[e];
          x[2 * e] = r;
        }
      } else if (c < 2 * n) {
        const float* cs = p.cos_sin + (long long)min(max(p.positions[tok[i]], 0), p.max_pos - 1) * p.rot_dims + (c < n ? c : c - n);
        const float sign = c < n ? -1.f : 1.f;
        const float4 c0 = *reinterpret_cast<const float4*>(cs), c1 = *reinterpret_cast<const float4*>(cs + 4);
        const float4 s0 = *reinterpret_cast<const float4*>(cs + n), s1 = *reinterpret_cast<const float4*>(cs + n + 4);
        const float cv[8] = {c0.x, c0.y, c0.z, c0.w, c1.x, c1.y, c1.z, c1.w};
        const float sv[8] = {s0.x, s0.y, s0.z, s0.w, s1.x, s1.y, s1.z, s1.w};
#pragma unroll
        for (int e = 0; e < 8; ++e) x[e] = x[e] * cv[e] + sign * y[e] * sv[e];
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) x[e] *= inv;
      dst = is_q ? reinterpret_cast<bf*>(p.q_out) + ((long long)tok[i] * p.a.heads + u) * p.a.dim_p
                 : reinterpret_cast<bf*>(p.k_cache) + ((blk * p.a.kv_heads + u - p.a.heads) * kMapsPage + off) * p.a.dim_p;
    }
    if (c < pad)
      *reinterpret_cast<uint4*>(dst + c) =
          make_uint4(pack_bf16x2(x[0], x[1]), pack_bf16x2(x[2], x[3]), pack_bf16x2(x[4], x[5]), pack_bf16x2(x[6], x[7]));
  }
}

template <int L>
static int launch_rope_norm_append8(const RopeNormAppendParams& p, long long warps, cudaStream_t s) {
  const long long per = 256 / L * kRopeUnits;
  return launch_pdl(rope_norm_append8_kernel<L>, dim3(unsigned((warps + per - 1) / per)), dim3(256), 0, s, p);
}

// ------------------------------------------------------------------------------------------------ simple
struct MapsSimpleParams {
  NkbMapsArgs a;
  const void *q, *k_cache, *v_cache;
  const int *block_table, *q_start, *q_lens, *context_lens;
  void* out;
  int batch, max_blocks;
};

constexpr int kSimpleWarps = 4;

// COLS: value columns per lane
template <typename T, int MAPS, int COLS>
__global__ void __launch_bounds__(kSimpleWarps * 32) maps_simple_kernel(const __grid_constant__ MapsSimpleParams p) {
  extern __shared__ float sm[];      // q [MAPS][dim_p], o [warps][MAPS][vdim_p], m [warps][MAPS], l [warps][MAPS], red[warps]
  const int t = blockIdx.x, h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kw = MAPS * p.a.dim_p, VP = p.a.vdim_p, v_ld = p.a.v_ld;
  float* q_s = sm;
  float* o_s = q_s + kw;
  float* m_s = o_s + kSimpleWarps * MAPS * VP;
  float* l_s = m_s + kSimpleWarps * MAPS;
  float* red = l_s + kSimpleWarps * MAPS;
  griddep_wait();
  griddep_launch();
  int b = -1, pos = 0;
  for (int i = 0; i < p.batch; ++i) {
    const int r = t - p.q_start[i];
    if (r >= 0 && r < p.q_lens[i]) {
      b = i;
      pos = p.context_lens[i] - p.q_lens[i] + r;
    }
  }
  T* out = reinterpret_cast<T*>(p.out) + t * p.a.o_token + h * p.a.o_head;
  if (b < 0 || pos < 0) {
    for (int c = threadIdx.x; c < p.a.vdim; c += blockDim.x) out[c] = cast_out<T>(0.f);
    return;
  }
  const T* q = reinterpret_cast<const T*>(p.q) + t * p.a.q_token + h * p.a.q_head;
  for (int c = threadIdx.x; c < kw; c += blockDim.x) q_s[c] = cast_in<T>(q[c]);
  __syncthreads();
  const int g = h / (p.a.heads / p.a.kv_heads);
  const int* table = p.block_table + (long long)b * p.max_blocks;
  float o[MAPS][COLS], m[MAPS], l[MAPS];
#pragma unroll
  for (int mp = 0; mp < MAPS; ++mp) {
    m[mp] = -INFINITY;
    l[mp] = 0.f;
#pragma unroll
    for (int i = 0; i < COLS; ++i) o[mp][i] = 0.f;
  }
  const int pages = pos / kMapsPage + 1;
  const int lo = nkb_first_visible(pos, p.a.window, p.a.chunk), page_lo = lo / kMapsPage;
  const int keep = p.a.keep_first, kept = min((keep + kMapsPage - 1) / kMapsPage, page_lo);   // pages of kept tokens before the window
  const float da = p.a.dist_a ? p.a.dist_a[h] : 0.f, db = p.a.dist_a ? p.a.dist_b[h] : 0.f;
  for (int i = warp; i < kept + pages - page_lo; i += kSimpleWarps) {
    const int pg = i < kept ? i : i - kept + page_lo;
    const long long blk = table[pg];
    const T* kr = reinterpret_cast<const T*>(p.k_cache) + ((blk * p.a.kv_heads + g) * kMapsPage + lane) * kw;
    const T* vb = reinterpret_cast<const T*>(p.v_cache) + (blk * p.a.kv_heads + g) * kMapsPage * v_ld;
    const int key = pg * kMapsPage + lane;
    const bool vis = key <= pos && (key >= lo || key < keep);
    const int nvis = min(kMapsPage, pos + 1 - pg * kMapsPage);
    float pr[MAPS];
#pragma unroll
    for (int mp = 0; mp < MAPS; ++mp) {
      float s = 0.f;
      if (vis) {
        for (int c = 0; c < p.a.dim; ++c) s = fmaf(q_s[mp * p.a.dim_p + c], cast_in<T>(kr[mp * p.a.dim_p + c]), s);
        s *= p.a.scale;
        if (p.a.softcap > 0.f) s = p.a.softcap * tanhf(s / p.a.softcap);
        if (p.a.dist_a) s -= da * log1pf(db * float(pos - key));
      } else {
        s = -INFINITY;
      }
      const float mn = fmaxf(m[mp], warp_max(s));            // finite: every page read holds a visible token
      const float alpha = expf(m[mp] - mn);
      pr[mp] = expf(s - mn);
      l[mp] = l[mp] * alpha + warp_sum(pr[mp]);
      m[mp] = mn;
#pragma unroll
      for (int i = 0; i < COLS; ++i) o[mp][i] *= alpha;
    }
    for (int j = 0; j < nvis; ++j) {
      float pj[MAPS];
#pragma unroll
      for (int mp = 0; mp < MAPS; ++mp) pj[mp] = __shfl_sync(0xffffffffu, pr[mp], j);
#pragma unroll
      for (int i = 0; i < COLS; ++i) {
        const int c = lane + 32 * i;
        if (c < VP) {
          const float v = cast_in<T>(vb[j * v_ld + c]);
#pragma unroll
          for (int mp = 0; mp < MAPS; ++mp) o[mp][i] = fmaf(pj[mp], v, o[mp][i]);
        }
      }
    }
  }
#pragma unroll
  for (int mp = 0; mp < MAPS; ++mp) {
#pragma unroll
    for (int i = 0; i < COLS; ++i)
      if (lane + 32 * i < VP) o_s[(warp * MAPS + mp) * VP + lane + 32 * i] = o[mp][i];
    if (lane == 0) {
      m_s[warp * MAPS + mp] = m[mp];
      l_s[warp * MAPS + mp] = l[mp];
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = threadIdx.x; c < p.a.vdim; c += blockDim.x) {
    float a[MAPS];
#pragma unroll
    for (int mp = 0; mp < MAPS; ++mp) {
      float mx = -INFINITY, acc = 0.f, den = 0.f;
      for (int w = 0; w < kSimpleWarps; ++w) mx = fmaxf(mx, m_s[w * MAPS + mp]);
      if (p.a.sinks) {
        mx = fmaxf(mx, p.a.sinks[h]);
        den = expf(p.a.sinks[h] - mx);
      }
      for (int w = 0; w < kSimpleWarps; ++w) {
        const float mw = m_s[w * MAPS + mp];
        const float f = mw == -INFINITY ? 0.f : expf(mw - mx);
        acc += f * o_s[(w * MAPS + mp) * VP + c];
        den += f * l_s[w * MAPS + mp];
      }
      a[mp] = acc / den;
    }
    const float r = MAPS == 2 ? a[0] - p.a.lambda * a[MAPS - 1] : a[0];
    ss += r * r;
    o_s[c] = r;                      // warp 0's map 0 slot of this column: read above by this thread only
  }
  if (MAPS == 2) {
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    float tot = 0.f;
    for (int w = 0; w < kSimpleWarps; ++w) tot += red[w];
    const float inv = p.a.out_scale / sqrtf(tot / float(p.a.vdim) + p.a.eps);
    for (int c = threadIdx.x; c < p.a.vdim; c += blockDim.x) out[c] = cast_out<T>(o_s[c] * inv);
  } else {
    for (int c = threadIdx.x; c < p.a.vdim; c += blockDim.x) out[c] = cast_out<T>(o_s[c]);
  }
}

// ------------------------------------------------------------------------------------------------ decode
constexpr int kMdStages = 3;
constexpr int kMdCounters = 16384;   // arrival counters in front of the split partials (as in attn_decode.cu)
constexpr int kMdHeads = 8;          // query heads of a CTA

struct MapsDecodeParams {
  NkbMapsArgs a;
  const __nv_bfloat16* q;
  const int *block_table, *context_lens;
  __nv_bfloat16* out;
  float* scratch;
  unsigned int* counters;
  int* status;
  int max_blocks, num_splits, chunks;    // chunks: groups of eight query heads per kv head
};

// base-2 logarithm domain score: optional cap, tanh written with the exponential (absolute error of an ulp or two
// of one, i.e. of the cap)
__device__ __forceinline__ float cap_score(float s, float scale, float cap, float inv_cap) {
  s *= scale;
  if (cap > 0.f) {
    const float e = exp2f(s * inv_cap * 2.885390081777927f);
    s = cap - 2.f * cap * __fdividef(1.f, e + 1.f);
  }
  return s * 1.4426950408889634f;
}

template <int KD, int VD, int W>
__global__ void __launch_bounds__(W * 32)
maps_decode_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV,
                   const __grid_constant__ MapsDecodeParams p) {
  constexpr int kSlab = kMapsPage * 128;     // 32 tokens x 64 columns
  constexpr int kKBytes = KD / 64 * kSlab, kVBytes = VD / 64 * kSlab, kStage = kKBytes + kVBytes;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  __shared__ uint64_t bars[W][kMdStages];
  __shared__ int abort_flag, is_last;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane >> 2, t = lane & 3;
  const int split = blockIdx.x, kvh = blockIdx.y / p.chunks, chunk = blockIdx.y % p.chunks, b = blockIdx.z;
  const int group = p.a.heads / p.a.kv_heads;
  const int head0 = kvh * group + chunk * kMdHeads, nh = min(kMdHeads, group - chunk * kMdHeads);
  if (threadIdx.x == 0) {
    for (int w = 0; w < W; ++w)
      for (int s = 0; s < kMdStages; ++s) mbar_init(&bars[w][s], 1);
    abort_flag = 0;
    mbar_fence_init();
    fence_proxy_async();
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
  }
  __syncthreads();
  griddep_wait();
  griddep_launch();
  const int ctx = p.context_lens[b];
  const int npages = ctx > 0 ? (ctx + kMapsPage - 1) / kMapsPage : 0;
  const int per_split = (npages + p.num_splits - 1) / p.num_splits;
  const int p0 = split * per_split, p1 = min(npages, p0 + per_split);
  const int* table = p.block_table + (long long)b * p.max_blocks;
  uint8_t* my_smem = smem + warp * kMdStages * kStage;
  auto issue = [&](int page, int stage) {
    if (lane == 0) {
      const int blk = table[page];
      uint8_t* dst = my_smem + stage * kStage;
      mbar_expect_tx(&bars[warp][stage], kStage);
#pragma unroll
      for (int h = 0; h < KD / 64; ++h) tma_load_4d(dst + h * kSlab, &tmK, &bars[warp][stage], h * 64, 0, kvh, blk);
#pragma unroll
      for (int h = 0; h < VD / 64; ++h)
        tma_load_4d(dst + kKBytes + h * kSlab, &tmV, &bars[warp][stage], h * 64, 0, kvh, blk);
    }
  };
  const int first = p0 + warp;
#pragma unroll
  for (int s = 0; s < kMdStages; ++s)
    if (first + s * W < p1) issue(first + s * W, s);

  // query fragments: rows g (map 0) and g + 8 (map 1) of query head head0 + g
  uint32_t qf[KD / 16][2];
  {
    const __nv_bfloat16* qr = p.q + ((long long)b * p.a.heads + head0 + g) * KD;
#pragma unroll
    for (int ks = 0; ks < KD / 16; ++ks) {
      qf[ks][0] = g < nh ? *reinterpret_cast<const uint32_t*>(qr + ks * 16 + 2 * t) : 0u;
      qf[ks][1] = g < nh ? *reinterpret_cast<const uint32_t*>(qr + ks * 16 + 8 + 2 * t) : 0u;
    }
  }
  const float inv_cap = p.a.softcap > 0.f ? 1.f / p.a.softcap : 0.f;
  float o[VD / 8][4];
#pragma unroll
  for (int i = 0; i < VD / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
  int stage = 0;
  uint32_t phase = 0;
  for (int pg = first; pg < p1; pg += W) {
    bool ok = mbar_wait(&bars[warp][stage], phase, &abort_flag, p.status, ERR_WAIT_SMEM_FULL);
    if (!__all_sync(0xffffffffu, ok)) break;
    const uint32_t kbase = smem_u32(my_smem + stage * kStage), vbase = kbase + kKBytes;
    float s[4][4];
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
#pragma unroll
    for (int kp = 0; kp < KD / 32; ++kp) {
      // contraction steps of the first half belong to map 0 (fragment rows 0-7), the others to map 1 (rows 8-15)
      const bool lo = kp < KD / 64;
      uint32_t a0[4], a1[4];
      a0[0] = lo ? qf[2 * kp][0] : 0u;     a0[1] = lo ? 0u : qf[2 * kp][0];
      a0[2] = lo ? qf[2 * kp][1] : 0u;     a0[3] = lo ? 0u : qf[2 * kp][1];
      a1[0] = lo ? qf[2 * kp + 1][0] : 0u; a1[1] = lo ? 0u : qf[2 * kp + 1][0];
      a1[2] = lo ? qf[2 * kp + 1][1] : 0u; a1[3] = lo ? 0u : qf[2 * kp + 1][1];
#pragma unroll
      for (int nt = 0; nt < 4; ++nt) {
        const int tok = nt * 8 + (lane & 7), ch = 4 * kp + (lane >> 3);
        const uint32_t addr = kbase + (ch >> 3) * kSlab + tok * 128 + (((ch & 7) ^ (tok & 7)) << 4);
        uint32_t b0, b1, b2, b3;
        ldsm_x4(addr, b0, b1, b2, b3);
        mma_16816(s[nt], a0, b0, b1);
        mma_16816(s[nt], a1, b2, b3);
      }
    }
    float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const bool vis = pg * kMapsPage + nt * 8 + 2 * t + e < ctx;
        const float v0 = vis ? cap_score(s[nt][e], p.a.scale, p.a.softcap, inv_cap) : -INFINITY;
        const float v1 = vis ? cap_score(s[nt][2 + e], p.a.scale, p.a.softcap, inv_cap) : -INFINITY;
        s[nt][e] = v0;
        s[nt][2 + e] = v1;
        mx0 = fmaxf(mx0, v0);
        mx1 = fmaxf(mx1, v1);
      }
    }
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
    const float n0 = fmaxf(m0, mx0), n1 = fmaxf(m1, mx1);     // finite: a page holds at least one visible token
    const float a0 = exp2f(m0 - n0), a1 = exp2f(m1 - n1);
    m0 = n0;
    m1 = n1;
    float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        s[nt][e] = exp2f(s[nt][e] - n0);
        s[nt][2 + e] = exp2f(s[nt][2 + e] - n1);
        sum0 += s[nt][e];
        sum1 += s[nt][2 + e];
      }
    }
    l0 = l0 * a0 + sum0;
    l1 = l1 * a1 + sum1;
#pragma unroll
    for (int i = 0; i < VD / 8; ++i) {
      o[i][0] *= a0; o[i][1] *= a0;
      o[i][2] *= a1; o[i][3] *= a1;
    }
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      uint32_t pa[4];
      pa[0] = pack_bf16x2(s[2 * j][0], s[2 * j][1]);
      pa[1] = pack_bf16x2(s[2 * j][2], s[2 * j][3]);
      pa[2] = pack_bf16x2(s[2 * j + 1][0], s[2 * j + 1][1]);
      pa[3] = pack_bf16x2(s[2 * j + 1][2], s[2 * j + 1][3]);
#pragma unroll
      for (int dp = 0; dp < VD / 16; ++dp) {
        const int tok = 16 * j + ((lane >> 3) & 1) * 8 + (lane & 7), ch = 2 * dp + (lane >> 4);
        const uint32_t addr = vbase + (ch >> 3) * kSlab + tok * 128 + (((ch & 7) ^ (tok & 7)) << 4);
        uint32_t v0, v1, v2, v3;
        ldsm_x4_t(addr, v0, v1, v2, v3);
        mma_16816(o[2 * dp], pa, v0, v1);
        mma_16816(o[2 * dp + 1], pa, v2, v3);
      }
    }
    __syncwarp();
    const int next = pg + kMdStages * W;
    if (next < p1) issue(next, stage);
    if (++stage == kMdStages) { stage = 0; phase ^= 1u; }
  }
  l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
  l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
  if (*(volatile int*)&abort_flag) {
    for (int i = 0; i < 200; ++i) __nanosleep(1000);
  }
  __syncthreads();     // every load consumed: the ring becomes merge space
  float* mo = reinterpret_cast<float*>(smem);      // [W][16][VD]
  float* mm = mo + W * 16 * VD;                    // [W][16]
  float* ml = mm + W * 16;                         // [W][16]
  float* fin = ml + W * 16;                        // [16][VD]
#pragma unroll
  for (int i = 0; i < VD / 8; ++i) {
    float* r0 = mo + (warp * 16 + g) * VD + i * 8 + 2 * t;
    float* r1 = r0 + 8 * VD;
    r0[0] = o[i][0]; r0[1] = o[i][1];
    r1[0] = o[i][2]; r1[1] = o[i][3];
  }
  if (t == 0) {
    mm[warp * 16 + g] = m0; mm[warp * 16 + g + 8] = m1;
    ml[warp * 16 + g] = l0; ml[warp * 16 + g + 8] = l1;
  }
  __syncthreads();
  const long long unit = (long long)b * gridDim.y + blockIdx.y;
  float* part = p.scratch + (unit * p.num_splits + split) * (16 * VD + 32);
  for (int idx = threadIdx.x; idx < 16 * VD; idx += W * 32) {
    const int r = idx / VD;
    float mf = -INFINITY;
#pragma unroll
    for (int w = 0; w < W; ++w) mf = fmaxf(mf, mm[w * 16 + r]);
    float acc = 0.f, l = 0.f;
#pragma unroll
    for (int w = 0; w < W; ++w) {
      const float mw = mm[w * 16 + r];
      const float sc = (mw == -INFINITY) ? 0.f : exp2f(mw - mf);
      acc += sc * mo[w * 16 * VD + idx];
      l += sc * ml[w * 16 + r];
    }
    if (p.num_splits == 1) {
      fin[idx] = l > 0.f ? acc / l : 0.f;
    } else {
      part[idx] = acc;
      if (idx % VD == 0) {
        part[16 * VD + r] = mf;
        part[16 * VD + 16 + r] = l;
      }
    }
  }
  if (p.num_splits > 1) {
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) {
      unsigned int* ctr = p.counters + unit;
      const unsigned int old = atomicAdd(ctr, 1u);
      is_last = old == unsigned(p.num_splits - 1);
      if (is_last) *ctr = 0u;
    }
    __syncthreads();
    if (!is_last) return;
    __threadfence();
    const float* base = p.scratch + unit * p.num_splits * (16 * VD + 32);
    for (int idx = threadIdx.x; idx < 16 * VD; idx += W * 32) {
      const int r = idx / VD;
      float mf = -INFINITY;
      for (int s = 0; s < p.num_splits; ++s) mf = fmaxf(mf, __ldcg(base + s * (16 * VD + 32) + 16 * VD + r));
      float acc = 0.f, l = 0.f;
      for (int s = 0; s < p.num_splits; ++s) {
        const float* ps = base + s * (16 * VD + 32);
        const float ms = __ldcg(ps + 16 * VD + r);
        const float sc = (ms == -INFINITY) ? 0.f : exp2f(ms - mf);
        acc += sc * __ldcg(ps + idx);
        l += sc * __ldcg(ps + 16 * VD + 16 + r);
      }
      fin[idx] = l > 0.f ? acc / l : 0.f;
    }
  }
  __syncthreads();
  for (int r = warp; r < nh; r += W) {
    float x[VD / 32], ss = 0.f;
#pragma unroll
    for (int i = 0; i < VD / 32; ++i) {
      x[i] = fin[r * VD + lane + 32 * i] - p.a.lambda * fin[(8 + r) * VD + lane + 32 * i];
      ss += x[i] * x[i];                            // padding columns hold zero
    }
    const float inv = p.a.out_scale / sqrtf(warp_sum(ss) / float(p.a.vdim) + p.a.eps);
    __nv_bfloat16* dst = p.out + ((long long)b * p.a.heads + head0 + r) * p.a.vdim;
#pragma unroll
    for (int i = 0; i < VD / 32; ++i)
      if (lane + 32 * i < p.a.vdim) dst[lane + 32 * i] = __float2bfloat16(x[i] * inv);
  }
}

template <int KD, int VD, int W>
static int launch_maps_decode(const CUtensorMap& tk, const CUtensorMap& tv, const MapsDecodeParams& p, int batch,
                              cudaStream_t s) {
  constexpr int kStage = (KD + VD) / 64 * kMapsPage * 128;
  constexpr int smem = W * kMdStages * kStage + 1024;
  static_assert(W * kMdStages * kStage >= int((W * 16 * VD + W * 32 + 16 * VD) * sizeof(float)), "merge space");
  static bool attr_set[64] = {false};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -1;
  if (!attr_set[dev]) {
    cudaError_t e = cudaFuncSetAttribute(maps_decode_kernel<KD, VD, W>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return int(e);
    attr_set[dev] = true;
  }
  return launch_pdl(maps_decode_kernel<KD, VD, W>, dim3(p.num_splits, p.a.kv_heads * p.chunks, batch), dim3(W * 32),
                    size_t(smem), s, tk, tv, p);
}
template <int KD, int VD>
static int maps_decode_warps(const CUtensorMap& tk, const CUtensorMap& tv, const MapsDecodeParams& p, int batch,
                             cudaStream_t s) {
  const long long ctas = (long long)batch * p.a.kv_heads * p.chunks * p.num_splits;
  if (ctas <= num_sms()) return launch_maps_decode<KD, VD, 4>(tk, tv, p, batch, s);
  if (ctas <= 2LL * num_sms()) return launch_maps_decode<KD, VD, 2>(tk, tv, p, batch, s);
  return launch_maps_decode<KD, VD, 1>(tk, tv, p, batch, s);
}

}  // namespace nkb

using namespace nkb;

static int maps_ok(const NkbMapsArgs& a) {
  return a.maps >= 1 && a.maps <= 2 && a.kv_heads >= 1 && a.heads >= a.kv_heads && a.heads % a.kv_heads == 0 && a.dim >= 2 &&
         a.dim_p >= a.dim && a.dim_p % 2 == 0 && a.vdim >= 1 && a.vdim_p >= a.vdim;
}

extern "C" int nkb_maps_append(const NkbMapsArgs* a, const NkbProj* q, const NkbProj* k, const NkbProj* v,
                               const float* cos_sin, int rot_dims, int max_pos, const int* positions, const int* slots,
                               void* q_out, void* k_cache, void* v_cache, int bf16, int tokens, int block_size,
                               void* stream) {
  if (tokens <= 0) return 0;
  if (!maps_ok(*a) || block_size != kMapsPage || rot_dims < 0 || rot_dims > a->dim || (rot_dims & 1) || max_pos < 1) return -2;
  MapsAppendParams p{};
  p.q = *q; p.k = *k; p.v = *v; p.a = *a;
  p.cos_sin = cos_sin; p.positions = positions; p.slots = slots;
  p.q_out = q_out; p.k_cache = k_cache; p.v_cache = v_cache;
  p.rot_dims = rot_dims; p.max_pos = max_pos; p.tokens = tokens;
  const auto al16 = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
  p.vec = ((a->dim | a->dim_p | a->vdim | a->vdim_p | rot_dims) & 3) == 0 && proj_vec4_ok(*q) && proj_vec4_ok(*k) &&
          proj_vec4_ok(*v) && al16(cos_sin) && al16(q_out) && al16(k_cache) && al16(v_cache);
  const long long warps = (long long)tokens * (a->heads + 2 * a->kv_heads);
  if (warps > 0x7fffffffll) return -2;
  const dim3 grid(unsigned((warps + 7) / 8));
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return bf16 ? launch_pdl(maps_append_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, p)
              : launch_pdl(maps_append_kernel<float>, grid, dim3(256), 0, s, p);
}

extern "C" int nkb_row_norm_append(const NkbMapsArgs* a, const NkbProj* q, const NkbProj* k, const NkbProj* v,
                                   const float* q_norm, const float* k_norm, const int* slots, void* q_out, void* k_cache,
                                   void* v_cache, int bf16, int tokens, int block_size, void* stream) {
  if (tokens <= 0) return 0;
  if (!maps_ok(*a) || a->maps != 1 || block_size != kMapsPage) return -2;
  RowNormAppendParams p{};
  p.q = *q; p.k = *k; p.v = *v; p.a = *a;
  p.q_norm = q_norm; p.k_norm = k_norm; p.slots = slots;
  p.q_out = q_out; p.k_cache = k_cache; p.v_cache = v_cache;
  const size_t smem = size_t(a->heads + a->kv_heads) * a->dim * sizeof(float);
  if (smem > 48 * 1024 - 128) return -2;
  const auto al16 = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
  const bool vec = ((a->dim | a->dim_p | a->vdim | a->vdim_p) & 3) == 0 && proj_vec4_ok(*q) && proj_vec4_ok(*k) &&
                   proj_vec4_ok(*v) && al16(q_out) && al16(k_cache) && al16(v_cache);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid(tokens), block(256);
  using bf = __nv_bfloat16;
  if (vec)
    return bf16 ? launch_pdl(row_norm_append_kernel<4, bf>, grid, block, smem, s, p)
                : launch_pdl(row_norm_append_kernel<4, float>, grid, block, smem, s, p);
  return bf16 ? launch_pdl(row_norm_append_kernel<1, bf>, grid, block, smem, s, p)
              : launch_pdl(row_norm_append_kernel<1, float>, grid, block, smem, s, p);
}

extern "C" int nkb_rope_norm_append(const NkbMapsArgs* a, const NkbProj* q, const NkbProj* k, const NkbProj* v,
                                    const float* bias, const float* cos_sin, int rot_dims, int max_pos, const int* positions,
                                    const int* slots, int norm, int pairs, void* q_out, void* k_cache, void* v_cache, int bf16, int tokens,
                                    int block_size, void* stream) {
  if (tokens <= 0) return 0;
  if (!maps_ok(*a) || a->maps != 1 || block_size != kMapsPage || rot_dims < 0 || rot_dims > a->dim || (rot_dims & 1) ||
      max_pos < 1 || (k->ptr && !v->ptr) || (rot_dims > 0 && !cos_sin))
    return -2;
  RopeNormAppendParams p{};
  p.q = *q; p.k = *k; p.v = *v; p.a = *a;
  p.bias = bias; p.cos_sin = cos_sin; p.positions = positions; p.slots = slots;
  p.q_out = q_out; p.k_cache = k_cache; p.v_cache = v_cache;
  p.rot_dims = rot_dims; p.max_pos = max_pos; p.tokens = tokens; p.norm = norm; p.pairs = pairs;
  const auto al16 = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
  // whole vectors on one side of the rotation's end (and, with halves, of its middle); angles in aligned runs
  const int half = pairs ? 1 : 2;
  const bool vec = ((a->dim | a->dim_p | a->vdim | a->vdim_p) & 3) == 0 && rot_dims % (4 * half) == 0 && proj_vec4_ok(*q) &&
                   proj_vec4_ok(*k) && proj_vec4_ok(*v) && al16(cos_sin) && al16(q_out) && al16(k_cache) && al16(v_cache);
  const long long warps = (long long)tokens * (a->heads + (k->ptr ? 2 * a->kv_heads : 0));
  if (warps > 0x7fffffffll) return -2;
  const dim3 grid(unsigned((warps + 7) / 8)), block(256);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  using bf = __nv_bfloat16;
  const auto whole = [&](const NkbProj& x) { return !x.ptr || (x.bf16 && al16(x.ptr) && (x.ld & 7) == 0); };
  const int wide = a->dim_p > a->vdim ? a->dim_p : a->vdim;
  if (bf16 && ((a->dim | a->dim_p | a->vdim | a->vdim_p) & 7) == 0 && rot_dims % (8 * half) == 0 && wide <= 256 && whole(*q) && whole(*k) &&
      whole(*v) && al16(q_out) && al16(k_cache) && al16(v_cache) && al16(bias) && al16(cos_sin)) {
    if (wide <= 64) return launch_rope_norm_append8<8>(p, warps, s);
    if (wide <= 128) return launch_rope_norm_append8<16>(p, warps, s);
    return launch_rope_norm_append8<32>(p, warps, s);
  }
  if (vec)
    return bf16 ? launch_pdl(rope_norm_append_kernel<4, bf>, grid, block, 0, s, p)
                : launch_pdl(rope_norm_append_kernel<4, float>, grid, block, 0, s, p);
  return bf16 ? launch_pdl(rope_norm_append_kernel<1, bf>, grid, block, 0, s, p)
              : launch_pdl(rope_norm_append_kernel<1, float>, grid, block, 0, s, p);
}

template <typename T>
static int launch_simple(const MapsSimpleParams& p, dim3 grid, size_t smem, cudaStream_t s) {
  const dim3 block(kSimpleWarps * 32);
  if (p.a.maps == 2)
    return p.a.vdim_p <= 256 ? launch_pdl(maps_simple_kernel<T, 2, 8>, grid, block, smem, s, p) : -2;
  if (p.a.vdim_p <= 256) return launch_pdl(maps_simple_kernel<T, 1, 8>, grid, block, smem, s, p);
  if (p.a.vdim_p <= 1024) return launch_pdl(maps_simple_kernel<T, 1, 32>, grid, block, smem, s, p);
  return -2;
}

extern "C" int nkb_maps_attn_simple(const NkbMapsArgs* a, const void* q, const void* k_cache, const void* v_cache,
                                    const int* block_table, const int* q_start, const int* q_lens,
                                    const int* context_lens, void* out, int bf16, int batch, int total_q, int block_size,
                                    int max_blocks_per_seq, void* stream) {
  if (batch <= 0 || total_q <= 0) return 0;
  if (!maps_ok(*a) || block_size != kMapsPage || a->heads > 65535 || ((a->sinks || a->dist_a || a->keep_first > 0) && a->maps != 1) ||
      a->keep_first < 0 || !a->dist_a != !a->dist_b)
    return -2;
  MapsSimpleParams p{};
  p.a = *a; p.q = q; p.k_cache = k_cache; p.v_cache = v_cache;
  p.block_table = block_table; p.q_start = q_start; p.q_lens = q_lens; p.context_lens = context_lens;
  p.out = out; p.batch = batch; p.max_blocks = max_blocks_per_seq;
  const int kw = a->maps * a->dim_p;
  if (!p.a.q_token) { p.a.q_token = (long long)a->heads * kw; p.a.q_head = kw; }
  if (!p.a.o_token) { p.a.o_token = (long long)a->heads * a->vdim; p.a.o_head = a->vdim; }
  if (!p.a.v_ld) p.a.v_ld = a->vdim_p;
  const size_t smem = size_t(kw + kSimpleWarps * (a->maps * a->vdim_p + 5)) * sizeof(float);
  if (smem > 48 * 1024) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid(total_q, a->heads);
  return bf16 ? launch_simple<__nv_bfloat16>(p, grid, smem, s) : launch_simple<float>(p, grid, smem, s);
}

extern "C" long long nkb_maps_decode_scratch_floats(const NkbMapsArgs* a, int batch, int num_splits) {
  if (num_splits <= 1) return 0;
  const int chunks = (a->heads / a->kv_heads + kMdHeads - 1) / kMdHeads;
  return kMdCounters + (long long)batch * a->kv_heads * chunks * num_splits * (16 * a->vdim_p + 32);
}

// One new token per sequence (row b of q / out = sequence b), already appended to the cache; two maps, bf16,
// dim_p 32 or 64, vdim_p 64 or 128.  Returns -5 for sizes it does not take.
extern "C" int nkb_maps_attn_decode(const NkbMapsArgs* a, const void* q, const void* k_cache, const void* v_cache,
                                    const int* block_table, const int* context_lens, void* out, float* scratch,
                                    int batch, int block_size, int num_blocks, int max_blocks_per_seq, int num_splits,
                                    void* stream) {
  if (batch <= 0) return 0;
  if (!maps_ok(*a) || block_size != kMapsPage || batch > 65535) return -2;
  if (a->maps != 2 || a->window > 0 || a->chunk > 0 || a->sinks || a->dist_a || (a->dim_p != 32 && a->dim_p != 64) || (a->vdim_p != 64 && a->vdim_p != 128)) return -5;
  if (!status_word() && nkb_init() != 0) return -1;
  MapsDecodeParams p{};
  p.a = *a;
  p.chunks = (a->heads / a->kv_heads + kMdHeads - 1) / kMdHeads;
  if (num_splits < 1) num_splits = 1;
  if (num_splits > 1 && (!scratch || (long long)batch * a->kv_heads * p.chunks > kMdCounters)) return -2;
  p.q = reinterpret_cast<const __nv_bfloat16*>(q);
  p.block_table = block_table; p.context_lens = context_lens;
  p.out = reinterpret_cast<__nv_bfloat16*>(out);
  p.scratch = num_splits > 1 ? scratch + kMdCounters : scratch;
  p.counters = reinterpret_cast<unsigned int*>(scratch);
  p.status = status_word();
  p.max_blocks = max_blocks_per_seq; p.num_splits = num_splits;
  const int kd = 2 * a->dim_p, vd = a->vdim_p;
  CUtensorMap tk, tv;
  const uint32_t box[4] = {64, uint32_t(kMapsPage), 1, 1};
  auto encode = [&](CUtensorMap* m, const void* ptr, int width) {
    const uint64_t dims[4] = {uint64_t(width), uint64_t(kMapsPage), uint64_t(a->kv_heads), uint64_t(num_blocks)};
    const uint64_t strides[3] = {uint64_t(width) * 2, uint64_t(width) * kMapsPage * 2,
                                 uint64_t(width) * kMapsPage * a->kv_heads * 2};
    return encode_tmap_bf16(m, ptr, 4, dims, strides, box);
  };
  if (encode(&tk, k_cache, kd) || encode(&tv, v_cache, vd)) return -4;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (kd == 64 && vd == 64) return maps_decode_warps<64, 64>(tk, tv, p, batch, s);
  if (kd == 64 && vd == 128) return maps_decode_warps<64, 128>(tk, tv, p, batch, s);
  if (kd == 128 && vd == 64) return maps_decode_warps<128, 64>(tk, tv, p, batch, s);
  return maps_decode_warps<128, 128>(tk, tv, p, batch, s);
}
