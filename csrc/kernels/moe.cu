// Mixture-of-experts token routing around the grouped expert GEMM: sort (token, expert)
// pairs by local expert, gather the token rows into expert-sorted order, and combine the
// weighted expert outputs per token.
//
// Reference parity: the reference evaluates MoE with per-token Python loops unrolled at
// trace time (examples/models/qwen3/kernels/transformer_layer.py:77-110) or by gathering the
// top-k expert matrices (examples/models/gpt_oss/kernels/feedforward.py:87-144), with every
// rank holding all experts.  Here experts are sharded over ranks (expert parallelism): a
// rank processes the pairs routed to its experts [expert_lo, expert_lo + num_local) and
// produces the partial sum of its experts' contributions for every token.
#include "common.cuh"
#include "api.h"

namespace nkb {

// counts[e] = number of pairs routed to local expert e
__global__ void moe_count_kernel(const int* __restrict__ experts, int pairs, int expert_lo, int num_local,
                                 int* __restrict__ counts) {
  griddep_wait();
  griddep_launch();
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= pairs) return;
  const int e = experts[i] - expert_lo;
  if (e >= 0 && e < num_local) atomicAdd(&counts[e], 1);
}

// exclusive scan of counts -> offsets[0..num_local], cursors reset to 0 (one block)
__global__ void moe_scan_kernel(const int* __restrict__ counts, int num_local, int* __restrict__ offsets,
                                int* __restrict__ cursors) {
  griddep_wait();
  griddep_launch();
  __shared__ int tmp[1024];
  const int t = threadIdx.x;
  tmp[t] = t < num_local ? counts[t] : 0;
  __syncthreads();
  for (int o = 1; o < 1024; o <<= 1) {
    const int v = t >= o ? tmp[t - o] : 0;
    __syncthreads();
    tmp[t] += v;
    __syncthreads();
  }
  if (t < num_local) {
    offsets[t + 1] = tmp[t];
    cursors[t] = 0;
  }
  if (t == 0) offsets[0] = 0;
}

// compact tile schedules for the grouped GEMMs: for tile width bn, group g contributes
// ceil(count_g / bn) tiles (one block; runs after the scan)
__global__ void moe_tiles_kernel(const int* __restrict__ offsets, int num_local, int bn_a, int* __restrict__ tiles_a,
                                 int* __restrict__ ntiles_a, int bn_b, int* __restrict__ tiles_b,
                                 int* __restrict__ ntiles_b) {
  griddep_wait();
  griddep_launch();
  __shared__ int sa[1024], sb[1024];
  const int t = threadIdx.x;
  const int n = t < num_local ? offsets[t + 1] - offsets[t] : 0;
  const int ca = (n + bn_a - 1) / bn_a, cb = (n + bn_b - 1) / bn_b;
  sa[t] = ca;
  sb[t] = cb;
  __syncthreads();
  for (int o = 1; o < 1024; o <<= 1) {
    const int va = t >= o ? sa[t - o] : 0, vb = t >= o ? sb[t - o] : 0;
    __syncthreads();
    sa[t] += va;
    sb[t] += vb;
    __syncthreads();
  }
  if (t < num_local) {
    int base = sa[t] - ca;
    for (int i = 0; i < ca; ++i) { tiles_a[2 * (base + i)] = t; tiles_a[2 * (base + i) + 1] = i; }
    base = sb[t] - cb;
    for (int i = 0; i < cb; ++i) { tiles_b[2 * (base + i)] = t; tiles_b[2 * (base + i) + 1] = i; }
  }
  if (t == 1023) { *ntiles_a = sa[1023]; *ntiles_b = sb[1023]; }
}

// Small batches (decode): one block counts, scans, assigns every pair its sorted position and
// builds both tile schedules, replacing the count / scan / tile kernels and the memset.
__global__ void moe_plan_small_kernel(const int* __restrict__ experts, int pairs, int expert_lo, int num_local,
                                      int* __restrict__ offsets, int* __restrict__ pair_pos,
                                      int* __restrict__ row_token, int top_k, int bn_a,
                                      int* __restrict__ tiles_a, int* __restrict__ ntiles_a, int bn_b,
                                      int* __restrict__ tiles_b, int* __restrict__ ntiles_b) {
  griddep_wait();
  griddep_launch();
  __shared__ int cnt[1024], off[1025], sa[1024], sb[1024];
  const int t = threadIdx.x;
  cnt[t] = 0;
  __syncthreads();
  for (int i = t; i < pairs; i += 1024) {
    const int e = experts[i] - expert_lo;
    if (e >= 0 && e < num_local) atomicAdd(&cnt[e], 1);
  }
  __syncthreads();
  const int n = t < num_local ? cnt[t] : 0;
  const int ca = (n + bn_a - 1) / bn_a, cb = (n + bn_b - 1) / bn_b;
  off[t + 1] = n;
  sa[t] = ca;
  sb[t] = cb;
  if (t == 0) off[0] = 0;
  __syncthreads();
  for (int o = 1; o < 1024; o <<= 1) {
    const int v = t >= o ? off[t + 1 - o] : 0, va = t >= o ? sa[t - o] : 0, vb = t >= o ? sb[t - o] : 0;
    __syncthreads();
    off[t + 1] += v;
    sa[t] += va;
    sb[t] += vb;
    __syncthreads();
  }
  if (t <= num_local) offsets[t] = off[t];
  if (t < num_local) {
    int base = sa[t] - ca;
    for (int i = 0; i < ca; ++i) { tiles_a[2 * (base + i)] = t; tiles_a[2 * (base + i) + 1] = i; }
    base = sb[t] - cb;
    for (int i = 0; i < cb; ++i) { tiles_b[2 * (base + i)] = t; tiles_b[2 * (base + i) + 1] = i; }
  }
  if (t == 1023) { *ntiles_a = sa[1023]; *ntiles_b = sb[1023]; }
  cnt[t] = 0;      // reused as per-expert cursors
  __syncthreads();
  // deterministic order inside an expert is not needed: every pair's output row is independent
  for (int i = t; i < pairs; i += 1024) {
    const int e = experts[i] - expert_lo;
    const int pos = (e >= 0 && e < num_local) ? off[e] + atomicAdd(&cnt[e], 1) : -1;
    pair_pos[i] = pos;
    if (row_token && pos >= 0) row_token[pos] = i / top_k;
  }
}

// The token row of a pair at its sorted position, multiplied by the pair's weight when there are weights (experts whose
// weight scales the input).
template <typename T>
__device__ __forceinline__ void moe_copy_row(const T* __restrict__ x, int hidden, int token, int pos, const float* pair_w,
                                             int pair, T* __restrict__ x_sorted) {
  const float w = pair_w ? pair_w[pair] : 1.f;
  const T* src = x + (long long)token * hidden;
  T* dst = x_sorted + (long long)pos * hidden;
  if constexpr (sizeof(T) == 4) {
    for (int v = threadIdx.x; v < hidden; v += blockDim.x) dst[v] = pair_w ? w * src[v] : src[v];
  } else if (hidden & 7) {
    for (int v = threadIdx.x; v < hidden; v += blockDim.x) dst[v] = __float2bfloat16(w * __bfloat162float(src[v]));
  } else {
    for (int v = threadIdx.x; v < (hidden >> 3); v += blockDim.x) {
      uint4 r = reinterpret_cast<const uint4*>(src)[v];
      if (pair_w) {
        uint32_t* rw = reinterpret_cast<uint32_t*>(&r);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 f = unpack_bf16x2(rw[e]);
          rw[e] = pack_bf16x2(w * f.x, w * f.y);
        }
      }
      reinterpret_cast<uint4*>(dst)[v] = r;
    }
  }
}

// one block per pair: copy the token row to its sorted position
template <typename T>
__global__ void moe_gather_kernel(const int* __restrict__ pair_pos, int top_k, const T* __restrict__ x, int hidden,
                                  const float* __restrict__ pair_w, T* __restrict__ x_sorted) {
  griddep_wait();
  griddep_launch();
  const int pair = blockIdx.x;
  const int pos = pair_pos[pair];
  if (pos >= 0) moe_copy_row<T>(x, hidden, pair / top_k, pos, pair_w, pair, x_sorted);
}

// one block per pair: claim a slot in its expert's segment and copy the token row there
template <typename T>
__global__ void moe_scatter_kernel(const int* __restrict__ experts, int pairs, int top_k, int expert_lo,
                                   int num_local, const int* __restrict__ offsets, int* __restrict__ cursors,
                                   const T* __restrict__ x, int hidden, const float* __restrict__ pair_w,
                                   T* __restrict__ x_sorted, int* __restrict__ pair_pos, int* __restrict__ row_token) {
  griddep_wait();
  griddep_launch();
  __shared__ int s_pos;
  const int pair = blockIdx.x;
  if (threadIdx.x == 0) {
    const int e = experts[pair] - expert_lo;
    int pos = -1;
    if (e >= 0 && e < num_local) pos = offsets[e] + atomicAdd(&cursors[e], 1);
    pair_pos[pair] = pos;
    if (row_token && pos >= 0) row_token[pos] = pair / top_k;
    s_pos = pos;
  }
  if (!x) return;
  __syncthreads();
  if (s_pos >= 0) moe_copy_row<T>(x, hidden, pair / top_k, s_pos, pair_w, pair, x_sorted);
}

// out[t] = sum_j w[t, j] * y_sorted[pair_pos[t * k + j]]   over the pairs handled locally
__global__ void moe_combine_kernel(const __nv_bfloat16* __restrict__ y_sorted, const int* __restrict__ pair_pos,
                                   const float* __restrict__ weights, int top_k, int hidden,
                                   __nv_bfloat16* __restrict__ out) {
  griddep_wait();
  griddep_launch();
  const int t = blockIdx.x;
  for (int v = threadIdx.x; v < (hidden >> 3); v += blockDim.x) {
    float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    for (int j = 0; j < top_k; ++j) {
      const int pos = pair_pos[t * top_k + j];
      if (pos < 0) continue;
      const float w = weights[t * top_k + j];
      const uint4 r = *reinterpret_cast<const uint4*>(y_sorted + (long long)pos * hidden + v * 8);
      const uint32_t rw[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 f = unpack_bf16x2(rw[e]);
        acc[2 * e] += w * f.x;
        acc[2 * e + 1] += w * f.y;
      }
    }
    uint4 o;
    o.x = pack_bf16x2(acc[0], acc[1]); o.y = pack_bf16x2(acc[2], acc[3]);
    o.z = pack_bf16x2(acc[4], acc[5]); o.w = pack_bf16x2(acc[6], acc[7]);
    *reinterpret_cast<uint4*>(out + (long long)t * hidden + v * 8) = o;
  }
}

}  // namespace nkb

using namespace nkb;

// experts [tokens * top_k] int32 (global expert ids).  Workspace (device, int32): counts[num_local],
// offsets[num_local + 1], cursors[num_local], pair_pos[tokens * top_k].  x_sorted must hold
// tokens * top_k rows.  After the call offsets / pair_pos / x_sorted are valid on the stream.  x == nullptr: the rows are
// not gathered (any width); row_token [tokens * top_k], when given, names the token of every sorted row instead.  pair_w
// [tokens * top_k]: the gathered rows are multiplied by it.  x_f32: x and x_sorted are fp32.
extern "C" int nkb_moe_dispatch(const int* experts, int tokens, int top_k, int expert_lo, int num_local, const void* x,
                                int x_f32, int hidden, const float* pair_w, void* x_sorted, int* counts, int* offsets, int* cursors, int* pair_pos,
                                int* row_token, int bn_a, int* tiles_a, int* ntiles_a, int bn_b, int* tiles_b, int* ntiles_b,
                                void* stream) {
  if (tokens <= 0) return 0;
  if (num_local > 1024 || (!x && !row_token) || bn_a <= 0 || bn_b <= 0) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const int pairs = tokens * top_k;
  if (pairs <= 8192) {
    int rc = launch_pdl(moe_plan_small_kernel, dim3(1), dim3(1024), 0, s, experts, pairs, expert_lo, num_local, offsets,
                        pair_pos, row_token, top_k, bn_a, tiles_a, ntiles_a, bn_b, tiles_b, ntiles_b);
    if (rc || !x) return rc;
    if (x_f32)
      return launch_pdl(moe_gather_kernel<float>, dim3(pairs), dim3(128), 0, s, (const int*)pair_pos, top_k,
                        (const float*)x, hidden, pair_w, (float*)x_sorted);
    return launch_pdl(moe_gather_kernel<__nv_bfloat16>, dim3(pairs), dim3(128), 0, s, (const int*)pair_pos, top_k,
                      (const __nv_bfloat16*)x, hidden, pair_w, (__nv_bfloat16*)x_sorted);
  }
  cudaError_t e = cudaMemsetAsync(counts, 0, sizeof(int) * num_local, s);
  if (e != cudaSuccess) return int(e);
  int rc = launch_pdl(moe_count_kernel, dim3((pairs + 255) / 256), dim3(256), 0, s, experts, pairs, expert_lo,
                      num_local, counts);
  if (rc) return rc;
  rc = launch_pdl(moe_scan_kernel, dim3(1), dim3(1024), 0, s, (const int*)counts, num_local, offsets, cursors);
  if (rc) return rc;
  rc = launch_pdl(moe_tiles_kernel, dim3(1), dim3(1024), 0, s, (const int*)offsets, num_local, bn_a, tiles_a, ntiles_a,
                  bn_b, tiles_b, ntiles_b);
  if (rc) return rc;
  if (x_f32)
    return launch_pdl(moe_scatter_kernel<float>, dim3(pairs), dim3(128), 0, s, experts, pairs, top_k, expert_lo, num_local,
                      (const int*)offsets, cursors, (const float*)x, hidden, pair_w, (float*)x_sorted, pair_pos, row_token);
  return launch_pdl(moe_scatter_kernel<__nv_bfloat16>, dim3(pairs), dim3(128), 0, s, experts, pairs, top_k, expert_lo, num_local,
                    (const int*)offsets, cursors, (const __nv_bfloat16*)x, hidden, pair_w, (__nv_bfloat16*)x_sorted, pair_pos,
                    row_token);
}

extern "C" int nkb_moe_combine(const void* y_sorted, const int* pair_pos, const float* weights, int tokens, int top_k,
                               int hidden, void* out, void* stream) {
  if (tokens <= 0) return 0;
  if (hidden & 7) return -2;
  return launch_pdl(moe_combine_kernel, dim3(tokens), dim3(256), 0, reinterpret_cast<cudaStream_t>(stream),
                    (const __nv_bfloat16*)y_sorted, pair_pos, weights, top_k, hidden, (__nv_bfloat16*)out);
}
