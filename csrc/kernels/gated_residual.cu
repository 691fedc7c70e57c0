// The elementwise ends of a layer whose residual stream stays in fp32:
//
//   embedding        x = table[id] * scale
//   residual         x <- x + sum_i branch_i   (+ a per-model vector) (+ a per-token matrix, both used ahead of a
//                    repeated block of layers); a branch is scaled, gated by sigmoid(gate_i + gate_bias_i) or by one gate
//                    per token, the weighted sum of the token's expert rows, or root-mean-square normed (NkbBranch)
//   group norms      out_j = w_j * x / sqrt(mean over the element's group of x^2 + eps), up to two weightings
//                    of one normalised row (layers whose two sublayers read the same residual); or layer norms
//                    w_j * (x - mean) / sqrt(variance + eps) + b_j; or plain copies of the row
//
// in one launch per layer: a CTA owns a token row, keeps it in shared memory between the sum and the norm, and
// takes the branches and gates as split-K partial sums, bf16 or fp32 (proj_src.h).  Also here: the activations
// act(gate) * up and act(x) over the same forms.
#include "common.cuh"
#include "proj_src.cuh"
#include "activations.cuh"
#include "api.h"

namespace nkb {

constexpr int kGrMaxGroups = 1024;
constexpr int kGrBranches = 3;
enum { NORM_RMS = 0, NORM_LAYER = 1, NORM_COPY = 2 };

struct GatedResidualParams {
  const float* x_in;              // fp32 rows, or nullptr with ids / table
  const int* ids;
  const void* table;              // [vocab, width], bf16 or fp32
  float scale;
  int vocab, table_bf16;
  int branches;
  NkbBranch br[kGrBranches];
  const float* add_row;           // [width] or nullptr
  const float* add_mat;           // [tokens, width] fp32 or nullptr
  float* x_out;                   // may be nullptr
  int norms, norm_kind;
  const float* w[2];
  const float* b[2];              // layer norms only
  void* out[2];
  int width, groups;
  float eps;
};

// Sum over the block; every thread gets it.  red: one float per warp, free again after the next barrier.
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < int(blockDim.x >> 5); ++i) t += red[i];
  return t;
}

template <int V>
__device__ __forceinline__ void load_vec(float (&a)[V], const float* p) {
  if constexpr (V == 4) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    a[0] = x.x; a[1] = x.y; a[2] = x.z; a[3] = x.w;
  } else {
    a[0] = *p;
  }
}
template <int V>
__device__ __forceinline__ void proj_vec(float (&a)[V], const NkbProj& s, long long row, int c) {
  if constexpr (V == 4) {
    const float4 x = proj_load4(s, row, c);
    a[0] = x.x; a[1] = x.y; a[2] = x.z; a[3] = x.w;
  } else {
    a[0] = proj_load(s, row, c);
  }
}

constexpr int kMaxTop = 32;

// Sum of a token's routed rows, four at a time so that their loads are in flight together; pos / w: the token's pairs.
template <int V>
__device__ __forceinline__ void pair_rows(float (&s)[V], const NkbBranch& br, const int* pos, const float* w, int c) {
  float a[V];
#pragma unroll
  for (int j = 0; j < V; ++j) a[j] = 0.f;
  if (V == 4 && br.y.bf16) {
    const __nv_bfloat16* y = reinterpret_cast<const __nv_bfloat16*>(br.y.ptr) + c;
#pragma unroll 1
    for (int i0 = 0; i0 < br.top_k; i0 += 4) {
      uint2 r[4];
#pragma unroll
      for (int i = 0; i < 4; ++i)
        r[i] = i0 + i < br.top_k ? *reinterpret_cast<const uint2*>(y + pos[i0 + i] * br.y.ld) : make_uint2(0u, 0u);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 lo = unpack_bf16x2(r[i].x), hi = unpack_bf16x2(r[i].y);
        const float x[4] = {lo.x, lo.y, hi.x, hi.y}, wi = i0 + i < br.top_k ? w[i0 + i] : 0.f;
#pragma unroll
        for (int j = 0; j < V; ++j) a[j] = fmaf(wi, x[j & 3], a[j]);
      }
    }
  } else {
#pragma unroll 1
    for (int i = 0; i < br.top_k; ++i) {
      float r[V];
      proj_vec<V>(r, br.y, pos[i], c);
#pragma unroll
      for (int j = 0; j < V; ++j) a[j] = fmaf(w[i], r[j], a[j]);
    }
  }
#pragma unroll
  for (int j = 0; j < V; ++j) s[j] = fmaf(br.scale, a[j], s[j]);
}

// What the branches of a launch are: all gated, all plain (scaled), one normed, or any mixture with routed ones.
enum { BR_GATED = 0, BR_PLAIN = 1, BR_ANY = 2, BR_NORMED = 3 };

// PACKED: every projection is bf16 and aligned (prefill), which keeps the kernel at few registers and many CTAs per SM
template <int V, bool PACKED, int MODE, typename OutT>
__global__ void __launch_bounds__(PACKED ? 256 : 1024, PACKED ? (MODE == BR_ANY ? 5 : 6) : 1)
gated_residual_kernel(const __grid_constant__ GatedResidualParams p) {
  extern __shared__ float row_s[];                 // [width] then [groups]
  __shared__ float red[32];
  float* inv_s = row_s + p.width;
  const long long t = blockIdx.x;
  const int nv = p.width / V;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  griddep_wait();
  griddep_launch();
  const int id = p.ids ? min(max(p.ids[t], 0), p.vocab - 1) : 0;
  __shared__ int pos_s[MODE == BR_ANY ? kGrBranches : 1][MODE == BR_ANY ? kMaxTop : 1];
  __shared__ float pw_s[MODE == BR_ANY ? kGrBranches : 1][MODE == BR_ANY ? kMaxTop : 1];
  __shared__ float tg_s[kGrBranches];
  float y_inv = 0.f;
  if constexpr (MODE == BR_NORMED) {
    float ss = 0.f;
    for (int i = threadIdx.x; i < nv; i += blockDim.x) {
      float y[V];
      proj_vec<V>(y, p.br[0].y, t, i * V);
#pragma unroll
      for (int j = 0; j < V; ++j) {
        ss += y[j] * y[j];
        row_s[i * V + j] = y[j];
      }
    }
    y_inv = p.br[0].scale / sqrtf(block_sum(ss, red) / float(p.width) + p.eps);
    __syncthreads();
  }
  if constexpr (MODE == BR_ANY) {
    // rows of pairs that are handled elsewhere count with weight zero (of a row that exists)
    for (int b = 0; b < p.branches; ++b) {
      if (p.br[b].token_gate && threadIdx.x == 0) tg_s[b] = sigmoid_f(proj_load(p.br[b].g, t, 0));
      if (p.br[b].pair_pos && int(threadIdx.x) < p.br[b].top_k) {
        const int pos = p.br[b].pair_pos[t * p.br[b].top_k + threadIdx.x];
        pos_s[b][threadIdx.x] = max(pos, 0);
        pw_s[b][threadIdx.x] = pos < 0 ? 0.f : p.br[b].pair_w ? p.br[b].pair_w[t * p.br[b].top_k + threadIdx.x] : 1.f;
      }
    }
    __syncthreads();
  }
  for (int i = threadIdx.x; i < nv; i += blockDim.x) {
    const int c = i * V;
    float a[V], s[V];
    if (p.x_in) {
      load_vec<V>(a, p.x_in + t * p.width + c);
    } else {
#pragma unroll
      for (int j = 0; j < V; ++j) {
        const long long o = (long long)id * p.width + c + j;
        a[j] = p.scale * (p.table_bf16 ? __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p.table)[o])
                                       : reinterpret_cast<const float*>(p.table)[o]);
      }
    }
#pragma unroll
    for (int j = 0; j < V; ++j) s[j] = 0.f;
    if constexpr (MODE == BR_ANY) {
#pragma unroll 1
      for (int b = 0; b < p.branches; ++b) {
        if (p.br[b].pair_pos) {
          pair_rows<V>(s, p.br[b], pos_s[b], pw_s[b], c);
          continue;
        }
        float y[V], w[V];
        proj_vec<V>(y, p.br[b].y, t, c);
#pragma unroll
        for (int j = 0; j < V; ++j) w[j] = p.br[b].scale;
        if (p.br[b].token_gate) {
#pragma unroll
          for (int j = 0; j < V; ++j) w[j] *= tg_s[b];
        } else if (p.br[b].g.ptr) {
          proj_vec<V>(w, p.br[b].g, t, c);
#pragma unroll
          for (int j = 0; j < V; ++j) w[j] = sigmoid_f(w[j] + p.br[b].gbias[c + j]);
        }
#pragma unroll
        for (int j = 0; j < V; ++j) s[j] = fmaf(w[j], y[j], s[j]);
      }
    } else if constexpr (MODE == BR_NORMED) {
      float w[V];
      load_vec<V>(w, p.br[0].norm_w + c);
#pragma unroll
      for (int j = 0; j < V; ++j) s[j] = row_s[c + j] * y_inv * w[j];
    } else if constexpr (PACKED) {
      uint2 y[2], g[2];
#pragma unroll
      for (int b = 0; b < 2; ++b)
        if (b < p.branches) {
          y[b] = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(p.br[b].y.ptr) + t * p.br[b].y.ld + c);
          if constexpr (MODE == BR_GATED)
            g[b] = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(p.br[b].g.ptr) + t * p.br[b].g.ld + c);
        }
#pragma unroll
      for (int b = 0; b < 2; ++b)
        if (b < p.branches) {
          const float2 y0 = unpack_bf16x2(y[b].x), y1 = unpack_bf16x2(y[b].y);
          if constexpr (MODE == BR_GATED) {
            const float4 bias = *reinterpret_cast<const float4*>(p.br[b].gbias + c);
            const float2 g0 = unpack_bf16x2(g[b].x), g1 = unpack_bf16x2(g[b].y);
            s[0] += y0.x * sigmoid_f(g0.x + bias.x);
            s[1] += y0.y * sigmoid_f(g0.y + bias.y);
            s[2] += y1.x * sigmoid_f(g1.x + bias.z);
            s[3] += y1.y * sigmoid_f(g1.y + bias.w);
          } else {
            const float w = p.br[b].scale;
            s[0] = fmaf(w, y0.x, s[0]);
            s[1] = fmaf(w, y0.y, s[1]);
            s[2] = fmaf(w, y1.x, s[2]);
            s[3] = fmaf(w, y1.y, s[3]);
          }
        }
    } else {
      float y[2][V], g[2][V];
#pragma unroll
      for (int b = 0; b < 2; ++b)
        if (b < p.branches) {
          proj_vec<V>(y[b], p.br[b].y, t, c);
          if constexpr (MODE == BR_GATED) proj_vec<V>(g[b], p.br[b].g, t, c);
        }
#pragma unroll
      for (int b = 0; b < 2; ++b)
        if (b < p.branches) {
          if constexpr (MODE == BR_GATED) {
            float bias[V];
            load_vec<V>(bias, p.br[b].gbias + c);
#pragma unroll
            for (int j = 0; j < V; ++j) s[j] += y[b][j] * sigmoid_f(g[b][j] + bias[j]);
          } else {
#pragma unroll
            for (int j = 0; j < V; ++j) s[j] = fmaf(p.br[b].scale, y[b][j], s[j]);
          }
        }
    }
#pragma unroll
    for (int j = 0; j < V; ++j) {
      a[j] += s[j];
      if (p.add_mat) a[j] += p.add_mat[t * p.width + c + j];
      if (p.add_row) a[j] += p.add_row[c + j];
    }
    if constexpr (V == 4) {
      *reinterpret_cast<float4*>(row_s + c) = make_float4(a[0], a[1], a[2], a[3]);
      if (p.x_out) *reinterpret_cast<float4*>(p.x_out + t * p.width + c) = make_float4(a[0], a[1], a[2], a[3]);
    } else {
      row_s[c] = a[0];
      if (p.x_out) p.x_out[t * p.width + c] = a[0];
    }
  }
  if (p.norms == 0) return;
  __syncthreads();
  const int gsz = p.width / p.groups;
  float mean = 0.f;
  if (p.norm_kind != NORM_RMS) {
    if (p.norm_kind == NORM_LAYER) {
      float a = 0.f, d2 = 0.f;
      for (int i = threadIdx.x; i < p.width; i += blockDim.x) a += row_s[i];
      mean = block_sum(a, red) / float(p.width);
      __syncthreads();
      for (int i = threadIdx.x; i < p.width; i += blockDim.x) {
        const float d = row_s[i] - mean;
        d2 += d * d;
      }
      d2 = block_sum(d2, red);
      if (threadIdx.x == 0) inv_s[0] = 1.f / sqrtf(d2 / float(p.width) + p.eps);
    } else if (threadIdx.x == 0) {
      inv_s[0] = 1.f;
    }
  } else if (p.groups <= nw) {
    // nw / groups warps share a group
    const int wpg = nw / p.groups, g = warp / wpg, sub = warp % wpg;
    float ss = 0.f;
    if (g < p.groups)
      for (int i = sub * 32 + lane; i < gsz; i += wpg * 32) {
        const float v = row_s[g * gsz + i];
        ss += v * v;
      }
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    if (int(threadIdx.x) < p.groups) {
      float tot = 0.f;
      for (int i = 0; i < wpg; ++i) tot += red[threadIdx.x * wpg + i];
      inv_s[threadIdx.x] = 1.f / sqrtf(tot / float(gsz) + p.eps);
    }
  } else {
    for (int g = warp; g < p.groups; g += nw) {
      float ss = 0.f;
      for (int i = lane; i < gsz; i += 32) {
        const float v = row_s[g * gsz + i];
        ss += v * v;
      }
      ss = warp_sum(ss);
      if (lane == 0) inv_s[g] = 1.f / sqrtf(ss / float(gsz) + p.eps);
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < nv; i += blockDim.x) {
    const int c = i * V;
    const float inv = inv_s[c / gsz];              // V > 1 only when a group is a multiple of V
    float a[V];
    load_vec<V>(a, row_s + c);
#pragma unroll
    for (int j = 0; j < V; ++j) a[j] = (a[j] - mean) * inv;
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      if (n < p.norms) {
        OutT* o = reinterpret_cast<OutT*>(p.out[n]) + t * p.width + c;
        float x[V];
#pragma unroll
        for (int j = 0; j < V; ++j) x[j] = a[j];
        if (p.w[n]) {
          float w[V];
          load_vec<V>(w, p.w[n] + c);
#pragma unroll
          for (int j = 0; j < V; ++j) x[j] *= w[j];
        }
        if (p.b[n]) {
          float w[V];
          load_vec<V>(w, p.b[n] + c);
#pragma unroll
          for (int j = 0; j < V; ++j) x[j] += w[j];
        }
        if constexpr (V == 4 && sizeof(OutT) == 2) {
          *reinterpret_cast<uint2*>(o) = make_uint2(pack_bf16x2(x[0], x[1]), pack_bf16x2(x[2], x[3]));
        } else {
#pragma unroll
          for (int j = 0; j < V; ++j) o[j] = cast_out<OutT>(x[j]);
        }
      }
    }
  }
}

// act(gate) * up, or act(gate) alone when up.ptr is null; up_rows: row up_rows[t] of up (a table of up_limit rows) instead
// of row t; ACT_CLAMPED: g sigmoid(alpha g) (u + 1) of g = min(gate, limit), u = clamp(up, -limit, limit); ACT_XIELU: its
// parameters are limit and alpha
template <int V, typename OutT>
__global__ void __launch_bounds__(256) gated_act_kernel(const __grid_constant__ NkbProj gate,
                                                        const __grid_constant__ NkbProj up, OutT* __restrict__ out,
                                                        int rows, int inter, int kind, float limit, float alpha,
                                                        const int* __restrict__ up_rows, int up_limit) {
  const int nv = inter / V;
  const long long n = (long long)rows * nv;
  griddep_wait();
  griddep_launch();
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / nv;
    const int c = int(i % nv) * V;
    float g[V], u[V];
    const long long ru = up_rows ? min(max(up_rows[r], 0), up_limit - 1) : r;
    if constexpr (V == 4) {
      const float4 a = proj_load4(gate, r, c);
      const float4 b = up.ptr ? proj_load4(up, ru, c) : make_float4(1.f, 1.f, 1.f, 1.f);
      g[0] = a.x; g[1] = a.y; g[2] = a.z; g[3] = a.w;
      u[0] = b.x; u[1] = b.y; u[2] = b.z; u[3] = b.w;
    } else {
      g[0] = proj_load(gate, r, c);
      u[0] = up.ptr ? proj_load(up, ru, c) : 1.f;
    }
    if (kind == ACT_CLAMPED) {
#pragma unroll
      for (int j = 0; j < V; ++j) {
        const float gc = fminf(g[j], limit), uc = fminf(fmaxf(u[j], -limit), limit);
        g[j] = gc / (1.f + expf(-alpha * gc)) * (uc + 1.f);
      }
    } else if (kind == ACT_XIELU) {
#pragma unroll
      for (int j = 0; j < V; ++j) g[j] = xielu(g[j], limit, alpha) * u[j];
    } else {
#pragma unroll
      for (int j = 0; j < V; ++j) g[j] = apply_act(g[j], kind) * u[j];
    }
    OutT* o = out + r * inter + c;
    if constexpr (V == 4 && sizeof(OutT) == 2) {
      *reinterpret_cast<uint2*>(o) = make_uint2(pack_bf16x2(g[0], g[1]), pack_bf16x2(g[2], g[3]));
    } else {
#pragma unroll
      for (int j = 0; j < V; ++j) o[j] = cast_out<OutT>(g[j]);
    }
  }
}

// Prompts: bf16 gate and up in whole 16-byte pieces, two pieces per thread in flight.
__global__ void __launch_bounds__(256) gated_act8_kernel(const __grid_constant__ NkbProj gate, const __grid_constant__ NkbProj up,
                                                         __nv_bfloat16* __restrict__ out, int pieces, int per_row, int kind,
                                                         float limit, float alpha) {
  griddep_wait();
  griddep_launch();
  uint4 g[2], u[2];
  int row[2], col[2];
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const int i = (blockIdx.x * 2 + k) * 256 + threadIdx.x;
    row[k] = i < pieces ? i / per_row : -1;
    col[k] = i < pieces ? i % per_row * 8 : 0;
    g[k] = u[k] = make_uint4(0u, 0u, 0u, 0u);
    if (row[k] >= 0) {
      g[k] = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(gate.ptr) + row[k] * gate.ld + col[k]);
      u[k] = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(up.ptr) + row[k] * up.ld + col[k]);
    }
  }
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    if (row[k] < 0) continue;
    const uint32_t gw[4] = {g[k].x, g[k].y, g[k].z, g[k].w}, uw[4] = {u[k].x, u[k].y, u[k].z, u[k].w};
    uint32_t r[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 a = unpack_bf16x2(gw[e]), b = unpack_bf16x2(uw[e]);
      float x[2] = {a.x, a.y}, y[2] = {b.x, b.y};
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        if (kind == ACT_CLAMPED) {
          x[j] = fminf(x[j], limit);
          x[j] *= sigmoid_f(alpha * x[j]) * (fminf(fmaxf(y[j], -limit), limit) + 1.f);
        } else {
          x[j] = apply_act(x[j], kind) * y[j];
        }
      }
      r[e] = pack_bf16x2(x[0], x[1]);
    }
    *reinterpret_cast<uint4*>(out + (long long)row[k] * per_row * 8 + col[k]) = make_uint4(r[0], r[1], r[2], r[3]);
  }
}

}  // namespace nkb

using namespace nkb;

static bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <int MODE>
static int launch_residual(const GatedResidualParams& p, bool packed, bool vec, int out_bf16, dim3 grid, dim3 block,
                           size_t smem, cudaStream_t s) {
  using bf = __nv_bfloat16;
  if (packed)
    return out_bf16 ? launch_pdl(gated_residual_kernel<4, true, MODE, bf>, grid, block, smem, s, p)
                    : launch_pdl(gated_residual_kernel<4, true, MODE, float>, grid, block, smem, s, p);
  if (vec)
    return out_bf16 ? launch_pdl(gated_residual_kernel<4, false, MODE, bf>, grid, block, smem, s, p)
                    : launch_pdl(gated_residual_kernel<4, false, MODE, float>, grid, block, smem, s, p);
  return out_bf16 ? launch_pdl(gated_residual_kernel<1, false, MODE, bf>, grid, block, smem, s, p)
                  : launch_pdl(gated_residual_kernel<1, false, MODE, float>, grid, block, smem, s, p);
}

extern "C" int nkb_gated_residual(const float* x_in, const int* ids, const void* table, int table_bf16, int vocab,
                                  float scale, int branches, const NkbBranch* br, const float* add_row,
                                  const float* add_mat, float* x_out, int norms, int norm_kind, const float* const* w,
                                  const float* const* b, void* const* out, int out_bf16, int rows, int width, int groups,
                                  float eps, void* stream) {
  if (rows <= 0) return 0;
  if (width <= 0 || width > 12000 || groups < 1 || groups > kGrMaxGroups || width % groups) return -2;
  if (norm_kind < NORM_RMS || norm_kind > NORM_COPY || (norm_kind != NORM_RMS && groups != 1)) return -2;
  if (branches < 0 || branches > kGrBranches || norms < 0 || norms > 2 || (!x_in && (!ids || !table || vocab < 1))) return -2;
  GatedResidualParams p{};
  p.x_in = x_in; p.ids = ids; p.table = table; p.scale = scale; p.vocab = vocab; p.table_bf16 = table_bf16;
  p.branches = branches; p.norms = norms; p.norm_kind = norm_kind;
  bool vec = width % 4 == 0 && (width / groups) % 4 == 0 && (!x_in || aligned16(x_in)) && (!x_out || aligned16(x_out));
  for (int i = 0; i < branches; ++i) {
    const NkbBranch& r = br[i];
    p.br[i] = r;
    if (r.pair_pos && (r.top_k < 1 || r.top_k > kMaxTop || r.g.ptr || r.norm_w)) return -2;
    if (r.norm_w && (branches != 1 || r.g.ptr)) return -2;
    if (r.token_gate ? !r.g.ptr || r.gbias : r.g.ptr && !r.gbias) return -2;
    vec = vec && proj_vec4_ok(r.y) && (r.token_gate || proj_vec4_ok(r.g)) && aligned16(r.gbias) && aligned16(r.norm_w);
  }
  for (int n = 0; n < norms; ++n) {
    p.w[n] = w[n]; p.b[n] = b ? b[n] : nullptr; p.out[n] = out[n];
    if (!w[n] && norm_kind != NORM_COPY) return -2;
    vec = vec && aligned16(w[n]) && aligned16(p.b[n]) && aligned16(out[n]);
  }
  p.add_row = add_row; p.add_mat = add_mat; p.x_out = x_out;
  p.width = width; p.groups = groups; p.eps = eps;
  const size_t smem = size_t(width + groups) * sizeof(float);
  bool packed = vec && branches > 0;
  for (int i = 0; i < branches; ++i) packed = packed && br[i].y.bf16 && (br[i].g.bf16 || !br[i].g.ptr || br[i].token_gate);
  // few rows: one vector per thread, so that every load of a row is in flight at once
  const int nv = vec ? width / 4 : width, most = packed || rows > 2 * 148 ? 256 : 1024;
  const int threads = nv >= most ? most : (nv < 64 ? 64 : (nv + 31) / 32 * 32);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (smem > 48 * 1024) return -2;
  const dim3 grid(rows), block(threads);
  int mode = BR_GATED;
  if (branches > 0) {
    int gated = 0, routed = 0;
    for (int i = 0; i < branches; ++i) {
      gated += br[i].g.ptr != nullptr;
      routed += br[i].pair_pos != nullptr || br[i].token_gate;
    }
    mode = br[0].norm_w ? BR_NORMED
           : routed || branches > 2 || (gated && gated < branches) ? BR_ANY : (gated ? BR_GATED : BR_PLAIN);
  }
  if (mode == BR_NORMED) return launch_residual<BR_NORMED>(p, packed, vec, out_bf16, grid, block, smem, s);
  if (mode == BR_GATED) return launch_residual<BR_GATED>(p, packed, vec, out_bf16, grid, block, smem, s);
  if (mode == BR_PLAIN) return launch_residual<BR_PLAIN>(p, packed, vec, out_bf16, grid, block, smem, s);
  return launch_residual<BR_ANY>(p, packed, vec, out_bf16, grid, block, smem, s);
}

extern "C" int nkb_gated_act(const NkbProj* gate, const NkbProj* up, void* out, int out_bf16, int rows, int inter,
                             int kind, float limit, float alpha, const int* up_rows, int up_limit, void* stream) {
  if (rows <= 0 || inter <= 0) return 0;
  if (kind < 0 || kind >= ACT_COUNT || (kind == ACT_CLAMPED && !up->ptr) || (up_rows && (!up->ptr || up_limit < 1))) return -2;
  const bool vec = inter % 4 == 0 && proj_vec4_ok(*gate) && proj_vec4_ok(*up) && aligned16(out);
  const long long n = (long long)rows * (vec ? inter / 4 : inter);
  const int blocks = int((n + 255) / 256 < 148 * 16 ? (n + 255) / 256 : 148 * 16);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  auto launch = [&](auto kernel, auto* o) {
    return launch_pdl(kernel, dim3(blocks), dim3(256), 0, s, *gate, *up, o, rows, inter, kind, limit, alpha, up_rows, up_limit);
  };
  using bf = __nv_bfloat16;
  const long long pieces = (long long)rows * (inter / 8);
  if (out_bf16 && kind != ACT_XIELU && gate->bf16 && up->ptr && up->bf16 && !up_rows && inter % 8 == 0 && ((gate->ld | up->ld) & 7) == 0 &&
      aligned16(gate->ptr) && aligned16(up->ptr) && aligned16(out) && pieces < (1ll << 30))
    return launch_pdl(gated_act8_kernel, dim3(unsigned((pieces + 511) / 512)), dim3(256), 0, s, *gate, *up, reinterpret_cast<bf*>(out),
                      int(pieces), inter / 8, kind, limit, alpha);
  if (out_bf16)
    return vec ? launch(gated_act_kernel<4, bf>, reinterpret_cast<bf*>(out)) : launch(gated_act_kernel<1, bf>, reinterpret_cast<bf*>(out));
  return vec ? launch(gated_act_kernel<4, float>, reinterpret_cast<float*>(out))
             : launch(gated_act_kernel<1, float>, reinterpret_cast<float*>(out));
}
