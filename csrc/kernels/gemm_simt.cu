// fp32-accumulating GEMM on the CUDA cores: out[m, n] = sum_k x[m, k] * w[n, k], operands fp32 or bf16, output fp32
// or bf16, any sizes and row strides.  Serves models that run in true 32-bit (no tensor-core mode keeps all 24
// mantissa bits) and the projections whose inner size has no 16-byte row pitch, which TMA cannot describe.
//
// A CTA of 256 threads owns a 64 x 64 tile of the output, four rows by four columns per thread; k-slabs of 16 are
// prefetched into registers while the previous slab is multiplied from shared memory.
#include "common.cuh"
#include "proj_src.cuh"
#include "api.h"

namespace nkb {

// The body of one tile: rows [m0, m) of x (through row_token when given) against rows of w.
template <typename XT, typename WT, typename OT>
__device__ __forceinline__ void simt_tile(const XT* __restrict__ x, const WT* __restrict__ w, OT* __restrict__ out, int m0,
                                          int m, int n0, int n, int k, long long ldx, long long ldw, long long ldo,
                                          const int* __restrict__ row_token) {
  constexpr int kT = 64, kK = 16;
  __shared__ __align__(16) float xs[kK][kT + 4], ws[kK][kT + 4];
  const int tr = threadIdx.x >> 4, tc = threadIdx.x & 15;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;   // loader: row, first of four k
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  float rx[4], rw[4];
  const long long xr = m0 + lr < m ? (row_token ? row_token[m0 + lr] : m0 + lr) : 0;
  auto fetch = [&](int k0) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int kk = k0 + lk + e;
      rx[e] = (m0 + lr < m && kk < k) ? cast_in<XT>(x[xr * ldx + kk]) : 0.f;
      rw[e] = (n0 + lr < n && kk < k) ? cast_in<WT>(w[(long long)(n0 + lr) * ldw + kk]) : 0.f;
    }
  };
  fetch(0);
  for (int k0 = 0; k0 < k; k0 += kK) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      xs[lk + e][lr] = rx[e];
      ws[lk + e][lr] = rw[e];
    }
    __syncthreads();
    if (k0 + kK < k) fetch(k0 + kK);
#pragma unroll
    for (int kk = 0; kk < kK; ++kk) {
      const float4 a = *reinterpret_cast<const float4*>(&xs[kk][tr * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&ws[kk][tc * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = m0 + tr * 4 + i;
    if (r >= m) break;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = n0 + tc * 4 + j;
      if (c < n) out[(long long)r * ldo + c] = cast_out<OT>(acc[i][j]);
    }
  }
}

template <typename XT, typename WT, typename OT>
__global__ void __launch_bounds__(256)
gemm_simt_kernel(const XT* __restrict__ x, const WT* __restrict__ w, OT* __restrict__ out, int m, int n, int k,
                 long long ldx, long long ldw, long long ldo) {
  griddep_wait();
  griddep_launch();
  simt_tile<XT, WT, OT>(x, w, out, blockIdx.y * 64, m, blockIdx.x * 64, n, k, ldx, ldw, ldo, nullptr);
}

// rows of group g: [offsets[g], offsets[g + 1]), weights w + g * n * k
template <typename XT, typename WT, typename OT>
__global__ void __launch_bounds__(256)
gemm_simt_grouped_kernel(const XT* __restrict__ x, const WT* __restrict__ w, OT* __restrict__ out,
                         const int* __restrict__ offsets, const int* __restrict__ row_token, int n, int k, long long ldx,
                         long long ldo) {
  griddep_wait();
  griddep_launch();
  const int g = blockIdx.z, m0 = offsets[g] + blockIdx.y * 64, m = offsets[g + 1];
  if (m0 >= m) return;
  simt_tile<XT, WT, OT>(x, w + (long long)g * n * k, out, m0, m, blockIdx.x * 64, n, k, ldx, k, ldo, row_token);
}

template <typename XT, typename WT, typename OT>
static int launch_simt(const void* x, const void* w, void* out, int m, int n, int k, long long ldx, long long ldw,
                       long long ldo, cudaStream_t s) {
  return launch_pdl(gemm_simt_kernel<XT, WT, OT>, dim3((n + 63) / 64, (m + 63) / 64), dim3(256), 0, s,
                    reinterpret_cast<const XT*>(x), reinterpret_cast<const WT*>(w), reinterpret_cast<OT*>(out), m, n, k,
                    ldx, ldw, ldo);
}
template <typename XT, typename WT, typename OT>
static int launch_simt_grouped(const void* x, const void* w, void* out, const int* offsets, const int* row_token,
                               int groups, int max_rows, int n, int k, long long ldx, long long ldo, cudaStream_t s) {
  return launch_pdl(gemm_simt_grouped_kernel<XT, WT, OT>, dim3((n + 63) / 64, (max_rows + 63) / 64, groups), dim3(256), 0, s,
                    reinterpret_cast<const XT*>(x), reinterpret_cast<const WT*>(w), reinterpret_cast<OT*>(out), offsets,
                    row_token, n, k, ldx, ldo);
}

}  // namespace nkb

using namespace nkb;

extern "C" int nkb_gemm_simt(const void* x, int x_bf16, const void* w, int w_bf16, void* out, int out_bf16, int m, int n,
                             int k, long long ldx, long long ldw, long long ldo, void* stream) {
  if (m <= 0 || n <= 0) return 0;
  if (k <= 0 || (m + 63) / 64 > 65535) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  using bf = __nv_bfloat16;
  if (!x_bf16 && !w_bf16 && !out_bf16) return launch_simt<float, float, float>(x, w, out, m, n, k, ldx, ldw, ldo, s);
  if (x_bf16 && w_bf16 && !out_bf16) return launch_simt<bf, bf, float>(x, w, out, m, n, k, ldx, ldw, ldo, s);
  if (x_bf16 && w_bf16 && out_bf16) return launch_simt<bf, bf, bf>(x, w, out, m, n, k, ldx, ldw, ldo, s);
  return -2;
}

// Rows sorted by group; row_token (may be null) names the row of x behind each sorted row.  w [groups, n, k].
extern "C" int nkb_gemm_simt_grouped(const void* x, int x_bf16, const void* w, int w_bf16, void* out, int out_bf16,
                                     const int* offsets, const int* row_token, int groups, int max_rows, int n, int k,
                                     long long ldx, long long ldo, void* stream) {
  if (groups <= 0 || max_rows <= 0 || n <= 0) return 0;
  if (k <= 0 || (max_rows + 63) / 64 > 65535 || groups > 65535) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  using bf = __nv_bfloat16;
  if (!x_bf16 && !w_bf16 && !out_bf16)
    return launch_simt_grouped<float, float, float>(x, w, out, offsets, row_token, groups, max_rows, n, k, ldx, ldo, s);
  if (x_bf16 && w_bf16 && !out_bf16)
    return launch_simt_grouped<bf, bf, float>(x, w, out, offsets, row_token, groups, max_rows, n, k, ldx, ldo, s);
  if (x_bf16 && w_bf16 && out_bf16)
    return launch_simt_grouped<bf, bf, bf>(x, w, out, offsets, row_token, groups, max_rows, n, k, ldx, ldo, s);
  return -2;
}
