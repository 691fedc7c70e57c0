// Residual update of layers that norm a sublayer's result before it is added, and of models whose layers read a weighted average of
// all earlier results (post_residual.h), in one launch.
//
// Everything is elementwise except the root mean squares of normed branches: those run with one CTA per token that keeps the
// branches' rows in shared memory between the sums and their use (NORMED); all others spread rows and columns freely.
#include "common.cuh"
#include "proj_src.cuh"
#include "post_residual.h"
#include "api.h"

namespace nkb {

// FAST: 1 - 2 / (exp(2 z) + 1) with the approximate exponential and reciprocal (errors of a few units in the last place of one),
// for results that are stored in bf16
template <bool FAST>
__device__ __forceinline__ float tanh_of(float z) {
  if constexpr (FAST) return 1.f - 2.f * __fdividef(1.f, __expf(2.f * z) + 1.f);
  return tanhf(z);
}

template <int V>
__device__ __forceinline__ void vec_in(float (&a)[V], const float* p) {
  if constexpr (V == 4) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    a[0] = x.x; a[1] = x.y; a[2] = x.z; a[3] = x.w;
  } else {
    a[0] = *p;
  }
}
template <int V>
__device__ __forceinline__ void vec_out(float* p, const float (&a)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(a[0], a[1], a[2], a[3]);
  else *p = a[0];
}
template <int V>
__device__ __forceinline__ void branch_in(float (&a)[V], const NkbPostBranch& br, long long t, int c) {
  if constexpr (V == 4) {
    const float4 x = proj_load4(br.y, t, c);
    a[0] = x.x; a[1] = x.y; a[2] = x.z; a[3] = x.w;
  } else {
    a[0] = proj_load(br.y, t, c);
  }
  if (br.shift) {
    float s[V];
    vec_in<V>(s, br.shift + c);
#pragma unroll
    for (int j = 0; j < V; ++j) a[j] += s[j];
  }
}

template <int V, bool FAST>
__device__ __forceinline__ void tanh_norm(float (&a)[V], const NkbTanhNorm& n, int c) {
  if (!n.w) return;
  float w[V], b[V];
  vec_in<V>(w, n.w + c);
  vec_in<V>(b, n.b + c);
#pragma unroll
  for (int j = 0; j < V; ++j) a[j] = fmaf(tanh_of<FAST>(n.alpha * a[j]), w[j], b[j]);
}

// What follows the sum s of the branches, for V elements of token t.
template <int V, typename OutT>
__device__ __forceinline__ void finish(const NkbPostResidual& p, float (&s)[V], float (&a)[V], long long t, int c) {
  constexpr bool FAST = sizeof(OutT) == 2;
  const long long o = t * p.width + c;
  if (p.branches) {
    tanh_norm<V, FAST>(s, p.post, c);
#pragma unroll
    for (int j = 0; j < V; ++j) a[j] += s[j];
  }
  if (p.result) vec_out<V>(p.result + o, a);
  if (p.coef) {
    const float last = p.coef[p.past];
#pragma unroll
    for (int j = 0; j < V; ++j) a[j] *= last;
    const float* h = p.history + o;
    int i = 0;
#pragma unroll 1
    for (; i + 4 <= p.past; i += 4) {                // four rows in flight
      float x[4][V];
#pragma unroll
      for (int k = 0; k < 4; ++k) vec_in<V>(x[k], h + (i + k) * p.history_stride);
#pragma unroll
      for (int k = 0; k < 4; ++k)
#pragma unroll
        for (int j = 0; j < V; ++j) a[j] = fmaf(p.coef[i + k], x[k][j], a[j]);
    }
#pragma unroll 1
    for (; i < p.past; ++i) {
      float x[V];
      vec_in<V>(x, h + i * p.history_stride);
#pragma unroll
      for (int j = 0; j < V; ++j) a[j] = fmaf(p.coef[i], x[j], a[j]);
    }
  }
  if (p.x_out) vec_out<V>(p.x_out + o, a);
#pragma unroll
  for (int n = 0; n < 2; ++n) {
    if (n >= p.norms) break;
    float x[V];
#pragma unroll
    for (int j = 0; j < V; ++j) x[j] = a[j];
    tanh_norm<V, FAST>(x, p.norm[n], c);
    OutT* out = reinterpret_cast<OutT*>(p.norm[n].out) + o;
    if constexpr (V == 4 && sizeof(OutT) == 2) {
      *reinterpret_cast<uint2*>(out) = make_uint2(pack_bf16x2(x[0], x[1]), pack_bf16x2(x[2], x[3]));
    } else {
#pragma unroll
      for (int j = 0; j < V; ++j) out[j] = cast_out<OutT>(x[j]);
    }
  }
}

template <int V>
__device__ __forceinline__ void stream_in(float (&a)[V], const NkbPostResidual& p, long long t, int c) {
  if (p.x_in) {
    vec_in<V>(a, p.x_in + t * p.width + c);
    return;
  }
  const long long o = (long long)min(max(p.ids[t], 0), p.vocab - 1) * p.width + c;
#pragma unroll
  for (int j = 0; j < V; ++j)
    a[j] = p.table_scale * (p.table_bf16 ? __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p.table)[o + j])
                                         : reinterpret_cast<const float*>(p.table)[o + j]);
}

template <int V, typename OutT>
__global__ void __launch_bounds__(256) post_residual_kernel(const __grid_constant__ NkbPostResidual p) {
  const long long t = blockIdx.y;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  griddep_wait();
  griddep_launch();
  for (long long r = t; r < p.rows; r += gridDim.y) {
    if (c >= p.width) return;
    float a[V], s[V];
    stream_in<V>(a, p, r, c);
#pragma unroll
    for (int j = 0; j < V; ++j) s[j] = 0.f;
#pragma unroll
    for (int b = 0; b < 2; ++b)
      if (b < p.branches) {
        float y[V];
        branch_in<V>(y, p.br[b], r, c);
#pragma unroll
        for (int j = 0; j < V; ++j) s[j] = fmaf(p.br[b].scale, y[j], s[j]);
      }
    finish<V, OutT>(p, s, a, r, c);
  }
}

// Normed branches (one with norm_w null is only scaled): a CTA per token.
template <int V, typename OutT>
__global__ void __launch_bounds__(1024) post_residual_normed_kernel(const __grid_constant__ NkbPostResidual p) {
  extern __shared__ __align__(16) float pr_s[];      // [branches][width]
  __shared__ float red[2][32];
  const long long t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  griddep_wait();
  griddep_launch();
  float ss[2] = {0.f, 0.f};
#pragma unroll
  for (int b = 0; b < 2; ++b)
    if (b < p.branches)
      for (int c = threadIdx.x * V; c < p.width; c += blockDim.x * V) {
        float y[V];
        branch_in<V>(y, p.br[b], t, c);
#pragma unroll
        for (int j = 0; j < V; ++j) ss[b] = fmaf(y[j], y[j], ss[b]);
        vec_out<V>(pr_s + b * p.width + c, y);
      }
#pragma unroll
  for (int b = 0; b < 2; ++b) {
    ss[b] = warp_sum(ss[b]);
    if (lane == 0) red[b][warp] = ss[b];
  }
  __syncthreads();
  float inv[2];
#pragma unroll
  for (int b = 0; b < 2; ++b) {
    float tot = 0.f;
    for (int w = 0; w < nw; ++w) tot += red[b][w];
    inv[b] = p.br[b].scale * (p.br[b].norm_w ? 1.f / sqrtf(tot / float(p.width) + p.eps) : 1.f);
  }
  for (int c = threadIdx.x * V; c < p.width; c += blockDim.x * V) {
    float a[V], s[V];
    stream_in<V>(a, p, t, c);
#pragma unroll
    for (int j = 0; j < V; ++j) s[j] = 0.f;
#pragma unroll
    for (int b = 0; b < 2; ++b)
      if (b < p.branches) {
        float y[V], w[V];
        vec_in<V>(y, pr_s + b * p.width + c);
#pragma unroll
        for (int j = 0; j < V; ++j) w[j] = 1.f;
        if (p.br[b].norm_w) vec_in<V>(w, p.br[b].norm_w + c);
#pragma unroll
        for (int j = 0; j < V; ++j) s[j] = fmaf(inv[b] * w[j], y[j], s[j]);
      }
    finish<V, OutT>(p, s, a, t, c);
  }
}

}  // namespace nkb

using namespace nkb;

extern "C" int nkb_post_residual(const NkbPostResidual* a, void* stream) {
  const NkbPostResidual& p = *a;
  if (p.rows <= 0) return 0;
  if (p.width <= 0 || p.width > 12000 || p.branches < 0 || p.branches > 2 || p.norms < 0 || p.norms > 2 || p.past < 0 ||
      (p.past > 0 && (!p.coef || !p.history)) || (!p.x_in && (!p.ids || !p.table || p.vocab < 1)))
    return -2;
  const auto al = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
  bool normed = false, vec = p.width % 4 == 0 && al(p.x_in) && al(p.result) && al(p.x_out) && al(p.history) &&
                             p.history_stride % 4 == 0 && al(p.post.w) && al(p.post.b);
  for (int i = 0; i < p.branches; ++i) {
    normed = normed || p.br[i].norm_w;
    vec = vec && proj_vec4_ok(p.br[i].y) && al(p.br[i].shift) && al(p.br[i].norm_w);
  }
  for (int n = 0; n < p.norms; ++n) {
    if (!p.norm[n].out || (p.norm[n].w && !p.norm[n].b)) return -2;
    vec = vec && al(p.norm[n].w) && al(p.norm[n].b) && al(p.norm[n].out);
  }
  if (p.post.w && !p.post.b) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const int nv = vec ? p.width / 4 : p.width;
  using bf = __nv_bfloat16;
  if (!normed) {
    const int threads = nv >= 256 ? 256 : (nv + 31) / 32 * 32;
    const dim3 grid((nv + threads - 1) / threads, p.rows < 65535 ? p.rows : 65535), block(threads);
    if (vec) return p.out_bf16 ? launch_pdl(post_residual_kernel<4, bf>, grid, block, 0, s, p)
                               : launch_pdl(post_residual_kernel<4, float>, grid, block, 0, s, p);
    return p.out_bf16 ? launch_pdl(post_residual_kernel<1, bf>, grid, block, 0, s, p)
                      : launch_pdl(post_residual_kernel<1, float>, grid, block, 0, s, p);
  }
  // few rows: one vector per thread, so that every load of a row is in flight at once
  const int most = p.rows > 2 * 148 ? 256 : 1024, threads = nv >= most ? most : (nv < 64 ? 64 : (nv + 31) / 32 * 32);
  const size_t smem = size_t(p.branches) * p.width * sizeof(float);
  auto launch = [&](auto kernel) {
    if (smem > 40 * 1024) {
      const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
      if (e != cudaSuccess) return int(e);
    }
    return launch_pdl(kernel, dim3(p.rows), dim3(threads), smem, s, p);
  };
  if (vec) return p.out_bf16 ? launch(post_residual_normed_kernel<4, bf>) : launch(post_residual_normed_kernel<4, float>);
  return p.out_bf16 ? launch(post_residual_normed_kernel<1, bf>) : launch(post_residual_normed_kernel<1, float>);
}
