// Latent attention (latent_attn.h) over a paged cache of latents:
//   append    the two down projections of a token: the query latent RMS-normed, the key / value latent RMS-normed and the
//             shared key part rotated (pairs 2i, 2i + 1) into the token's cache row
//   queries   the up-projected queries split into their unrotated and rotated parts, the latter rotated
//   gather    cached rows of whole pages as two matrices, the operands of the up projections of keys and values
//   attention any new tokens against the cached rows themselves, bf16: see latent_attn_kernel
#include "common.cuh"
#include "proj_src.cuh"
#include "latent_attn.h"
#include "attn_maps.h"
#include "api.h"
#include <math.h>

namespace nkb {

constexpr int kLatPage = 32;

template <typename T>
__device__ __forceinline__ void put(T* dst, const float (&x)[1]) { *dst = cast_out<T>(x[0]); }
template <typename T>
__device__ __forceinline__ void put(T* dst, const float (&x)[4]) {
  if constexpr (sizeof(T) == 2)
    *reinterpret_cast<uint2*>(dst) = make_uint2(pack_bf16x2(x[0], x[1]), pack_bf16x2(x[2], x[3]));
  else
    *reinterpret_cast<float4*>(dst) = make_float4(x[0], x[1], x[2], x[3]);
}
template <int V>
__device__ __forceinline__ void get(float (&x)[V], const NkbProj& s, long long row, int c) {
  if constexpr (V == 4) {
    const float4 r = proj_load4(s, row, c);
    x[0] = r.x; x[1] = r.y; x[2] = r.z; x[3] = r.w;
  } else {
    x[0] = proj_load(s, row, c);
  }
}
template <int V>
__device__ __forceinline__ void zero(float (&x)[V]) {
#pragma unroll
  for (int j = 0; j < V; ++j) x[j] = 0.f;
}
// V consecutive elements from column c of a rotated part of n pairs (2i, 2i + 1); cs: cosines, then sines of the n angles
template <int V>
__device__ __forceinline__ void rotate_pairs(float (&x)[V], const NkbProj& s, long long row, int col, int c, const float* cs,
                                             int n) {
  if constexpr (V == 4) {
    get<4>(x, s, row, col + c);
#pragma unroll
    for (int j = 0; j < 4; j += 2) {
      const float co = cs[(c + j) / 2], si = cs[n + (c + j) / 2], u = x[j], w = x[j + 1];
      x[j] = u * co - w * si;
      x[j + 1] = w * co + u * si;
    }
  } else {
    const int i = c / 2;
    const float u = proj_load(s, row, col + 2 * i), w = proj_load(s, row, col + 2 * i + 1);
    x[0] = (c & 1) ? w * cs[i] + u * cs[n + i] : u * cs[i] - w * cs[n + i];
  }
}

// ------------------------------------------------------------------------------------------------ append
struct LatentAppendParams {
  NkbProj q, kv;            // [q_rank], [rank + rot] columns
  NkbLatentArgs a;
  const float *q_norm, *kv_norm, *cos_sin;
  const int *positions, *slots;
  void *q_out, *cache;      // [tokens, q_rank], [blocks, 32, row]
  int max_pos;
};

template <int V, typename T>
__global__ void __launch_bounds__(256) latent_append_kernel(const __grid_constant__ LatentAppendParams p) {
  extern __shared__ __align__(16) float la_s[];     // query latent, key / value latent (at a multiple of four)
  __shared__ float red[2][8];
  const long long t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* kv_s = la_s + (p.a.q_rank + 3) / 4 * 4;
  griddep_wait();
  griddep_launch();
  float sq = 0.f, sk = 0.f;
  for (int c = threadIdx.x * V; c < p.a.q_rank; c += 256 * V) {
    float x[V];
    get<V>(x, p.q, t, c);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      sq += x[j] * x[j];
      la_s[c + j] = x[j];
    }
  }
  for (int c = threadIdx.x * V; c < p.a.rank; c += 256 * V) {
    float x[V];
    get<V>(x, p.kv, t, c);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      sk += x[j] * x[j];
      kv_s[c + j] = x[j];
    }
  }
  const int slot = p.slots[t];
  T* row = reinterpret_cast<T*>(p.cache) + (slot < 0 ? 0ll : (long long)slot) * p.a.row;   // pages follow one another
  if (slot >= 0) {
    const int pos = min(max(p.positions[t], 0), p.max_pos - 1);
    const float* cs = p.cos_sin + (long long)pos * p.a.rot;
    for (int c = threadIdx.x * V; c < p.a.row - p.a.rank; c += 256 * V) {
      float x[V];
      zero<V>(x);
      if (c < p.a.rot) rotate_pairs<V>(x, p.kv, t, p.a.rank, c, cs, p.a.rot / 2);
      put<T>(row + p.a.rank + c, x);
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
  const float iq = 1.f / sqrtf(tq / float(p.a.q_rank) + p.a.eps), ik = 1.f / sqrtf(tk / float(p.a.rank) + p.a.eps);
  T* qo = reinterpret_cast<T*>(p.q_out) + t * p.a.q_rank;
  for (int c = threadIdx.x * V; c < p.a.q_rank; c += 256 * V) {
    float x[V];
#pragma unroll
    for (int j = 0; j < V; ++j) x[j] = la_s[c + j] * iq * p.q_norm[c + j];
    put<T>(qo + c, x);
  }
  if (slot < 0) return;
  for (int c = threadIdx.x * V; c < p.a.rank; c += 256 * V) {
    float x[V];
#pragma unroll
    for (int j = 0; j < V; ++j) x[j] = kv_s[c + j] * ik * p.kv_norm[c + j];
    put<T>(row + c, x);
  }
}

__device__ __forceinline__ void unpack8(float (&x)[8], uint4 r) {
  const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const float2 f = unpack_bf16x2(w[e]);
    x[2 * e] = f.x;
    x[2 * e + 1] = f.y;
  }
}
__device__ __forceinline__ uint4 pack8(const float (&x)[8]) {
  return make_uint4(pack_bf16x2(x[0], x[1]), pack_bf16x2(x[2], x[3]), pack_bf16x2(x[4], x[5]), pack_bf16x2(x[6], x[7]));
}
__device__ __forceinline__ void load8(float (&x)[8], const float* p) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w;
  x[4] = b.x; x[5] = b.y; x[6] = b.z; x[7] = b.w;
}
// eight elements (four pairs) from column c of a rotated part of n pairs
__device__ __forceinline__ void rotate8(float (&x)[8], int c, const float* cs, int n) {
  const float4 co = *reinterpret_cast<const float4*>(cs + c / 2), si = *reinterpret_cast<const float4*>(cs + n + c / 2);
  const float cv[4] = {co.x, co.y, co.z, co.w}, sv[4] = {si.x, si.y, si.z, si.w};
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float u = x[2 * j], w = x[2 * j + 1];
    x[2 * j] = u * cv[j] - w * sv[j];
    x[2 * j + 1] = w * cv[j] + u * sv[j];
  }
}

// Prompts in bf16, sizes of whole 16-byte pieces: one warp per token, all of its loads in flight first.
constexpr int kAppendQ = 8, kAppendK = 4;            // pieces of a latent per lane: q_rank <= 2048, rank <= 1024

__global__ void __launch_bounds__(256) latent_append8_kernel(const __grid_constant__ LatentAppendParams p, int tokens) {
  using bf = __nv_bfloat16;
  const int t = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  griddep_wait();
  griddep_launch();
  if (t >= tokens) return;
  const bf* qs = reinterpret_cast<const bf*>(p.q.ptr) + t * p.q.ld;
  const bf* ks = reinterpret_cast<const bf*>(p.kv.ptr) + t * p.kv.ld;
  const int slot = p.slots[t], pos = min(max(p.positions[t], 0), p.max_pos - 1);
  uint4 q[kAppendQ], k[kAppendK], r = make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
  for (int i = 0; i < kAppendQ; ++i) {
    const int c = (i * 32 + lane) * 8;
    q[i] = c < p.a.q_rank ? *reinterpret_cast<const uint4*>(qs + c) : make_uint4(0u, 0u, 0u, 0u);
  }
#pragma unroll
  for (int i = 0; i < kAppendK; ++i) {
    const int c = (i * 32 + lane) * 8;
    k[i] = c < p.a.rank ? *reinterpret_cast<const uint4*>(ks + c) : make_uint4(0u, 0u, 0u, 0u);
  }
  if (lane * 8 < p.a.rot) r = *reinterpret_cast<const uint4*>(ks + p.a.rank + lane * 8);
  const auto squares = [](uint4 v) {
    float x[8], s = 0.f;
    unpack8(x, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) s += x[j] * x[j];
    return s;
  };
  float sq = 0.f, sk = 0.f;
#pragma unroll
  for (int i = 0; i < kAppendQ; ++i) sq += squares(q[i]);
#pragma unroll
  for (int i = 0; i < kAppendK; ++i) sk += squares(k[i]);
  const float iq = 1.f / sqrtf(warp_sum(sq) / float(p.a.q_rank) + p.a.eps);
  const float ik = 1.f / sqrtf(warp_sum(sk) / float(p.a.rank) + p.a.eps);
  const auto scaled = [](uint4 v, float inv, const float* w) {
    float x[8], ww[8];
    unpack8(x, v);
    load8(ww, w);
#pragma unroll
    for (int j = 0; j < 8; ++j) x[j] *= inv * ww[j];
    return pack8(x);
  };
  bf* qo = reinterpret_cast<bf*>(p.q_out) + (long long)t * p.a.q_rank;
#pragma unroll
  for (int i = 0; i < kAppendQ; ++i) {
    const int c = (i * 32 + lane) * 8;
    if (c < p.a.q_rank) *reinterpret_cast<uint4*>(qo + c) = scaled(q[i], iq, p.q_norm + c);
  }
  if (slot < 0) return;
  bf* row = reinterpret_cast<bf*>(p.cache) + (long long)slot * p.a.row;
#pragma unroll
  for (int i = 0; i < kAppendK; ++i) {
    const int c = (i * 32 + lane) * 8;
    if (c < p.a.rank) *reinterpret_cast<uint4*>(row + c) = scaled(k[i], ik, p.kv_norm + c);
  }
  if (lane * 8 < p.a.row - p.a.rank) {
    float x[8];
    unpack8(x, r);
    if (lane * 8 < p.a.rot) rotate8(x, lane * 8, p.cos_sin + (long long)pos * p.a.rot, p.a.rot / 2);
    *reinterpret_cast<uint4*>(row + p.a.rank + lane * 8) = pack8(x);
  }
}

// ------------------------------------------------------------------------------------------------ queries
struct LatentQueryParams {
  NkbProj q;                // [tokens, heads * (dim + rot)]
  NkbLatentArgs a;
  const float* cos_sin;
  const int* positions;
  void *plain, *rotated;    // element strides below; both padded with zeros to plain_pad / rot_pad elements
  long long plain_token, plain_head, rot_token, rot_head, rows;
  int plain_pad, rot_pad, max_pos;
};

template <int V, typename T>
__global__ void __launch_bounds__(256) latent_query_kernel(const __grid_constant__ LatentQueryParams p) {
  const long long gw = (blockIdx.x * 256ll + threadIdx.x) >> 5;
  const int lane = threadIdx.x & 31;
  griddep_wait();
  griddep_launch();
  if (gw >= p.rows) return;
  const int t = int(unsigned(gw) / unsigned(p.a.heads)), h = int(unsigned(gw) % unsigned(p.a.heads));
  const int col = h * (p.a.dim + p.a.rot);
  T* plain = reinterpret_cast<T*>(p.plain) + t * p.plain_token + h * p.plain_head;
  T* rotated = reinterpret_cast<T*>(p.rotated) + t * p.rot_token + h * p.rot_head;
  const float* cs = p.cos_sin + (long long)min(max(p.positions[t], 0), p.max_pos - 1) * p.a.rot;
  for (int i = lane * V; i < p.plain_pad + p.rot_pad; i += 32 * V) {
    float x[V];
    zero<V>(x);
    if (i < p.plain_pad) {
      if (i < p.a.dim) get<V>(x, p.q, t, col + i);
      put<T>(plain + i, x);
    } else {
      const int c = i - p.plain_pad;
      if (c < p.a.rot) rotate_pairs<V>(x, p.q, t, col + p.a.dim, c, cs, p.a.rot / 2);
      put<T>(rotated + c, x);
    }
  }
}

// Prompts in bf16, sizes of whole 16-byte pieces: one CTA per token, kQueryUnroll pieces per thread in flight.
constexpr int kQueryUnroll = 4;

__global__ void __launch_bounds__(256) latent_query8_kernel(const __grid_constant__ LatentQueryParams p) {
  using bf = __nv_bfloat16;
  const long long t = blockIdx.x;
  const int per = (p.plain_pad + p.rot_pad) / 8, n = p.a.heads * per;
  griddep_wait();
  griddep_launch();
  const bf* src = reinterpret_cast<const bf*>(p.q.ptr) + t * p.q.ld;
  bf* plain = reinterpret_cast<bf*>(p.plain) + t * p.plain_token;
  bf* rotated = reinterpret_cast<bf*>(p.rotated) + t * p.rot_token;
  const float* cs = p.cos_sin + (long long)min(max(p.positions[t], 0), p.max_pos - 1) * p.a.rot;
  for (int i0 = threadIdx.x; i0 < n; i0 += 256 * kQueryUnroll) {
    uint4 r[kQueryUnroll];
    int hd[kQueryUnroll], col[kQueryUnroll];
#pragma unroll
    for (int u = 0; u < kQueryUnroll; ++u) {
      const int i = i0 + u * 256;
      hd[u] = i / per;
      col[u] = (i % per) * 8;
      r[u] = make_uint4(0u, 0u, 0u, 0u);
      const bool rot = col[u] >= p.plain_pad;
      const int c = rot ? col[u] - p.plain_pad : col[u];
      if (i < n && c < (rot ? p.a.rot : p.a.dim))
        r[u] = *reinterpret_cast<const uint4*>(src + hd[u] * (p.a.dim + p.a.rot) + (rot ? p.a.dim : 0) + c);
    }
#pragma unroll
    for (int u = 0; u < kQueryUnroll; ++u) {
      if (i0 + u * 256 >= n) break;
      if (col[u] < p.plain_pad) {
        *reinterpret_cast<uint4*>(plain + hd[u] * p.plain_head + col[u]) = r[u];
        continue;
      }
      const int c = col[u] - p.plain_pad;
      if (c < p.a.rot) {
        float x[8];
        unpack8(x, r[u]);
        rotate8(x, c, cs, p.a.rot / 2);
        r[u] = pack8(x);
      }
      *reinterpret_cast<uint4*>(rotated + hd[u] * p.rot_head + c) = r[u];
    }
  }
}

// ------------------------------------------------------------------------------------------------ gather
// One CTA per page: cached rows -> latents [.., rank] and rotated parts [.., rot_ld] (padding of the cache row included).
template <typename T>
__global__ void __launch_bounds__(256) latent_gather_kernel(const T* __restrict__ cache, const int* __restrict__ pages, int row,
                                                            int rank, int rot, int rot_ld, T* __restrict__ c_out,
                                                            T* __restrict__ r_out) {
  griddep_wait();
  griddep_launch();
  constexpr int V = 16 / sizeof(T);
  const long long page = pages[blockIdx.x];
  const T* src = cache + page * kLatPage * row;
  const long long dst = (long long)blockIdx.x * kLatPage;
  if (rank % V == 0 && rot % V == 0 && rot_ld % V == 0) {
    const int per = (rank + rot) / V;
    for (int i = threadIdx.x; i < kLatPage * per; i += 256) {
      const int r = i / per, c = (i % per) * V;
      const uint4 x = *reinterpret_cast<const uint4*>(src + r * row + c);
      *reinterpret_cast<uint4*>(c < rank ? c_out + (dst + r) * rank + c : r_out + (dst + r) * rot_ld + c - rank) = x;
    }
  } else {
    for (int i = threadIdx.x; i < kLatPage * (rank + rot); i += 256) {
      const int r = i / (rank + rot), c = i % (rank + rot);
      (c < rank ? c_out[(dst + r) * rank + c] : r_out[(dst + r) * rot_ld + c - rank]) = src[r * row + c];
    }
  }
}

// ------------------------------------------------------------------------------------------------ attention
// One CTA per (split of the visible pages, N heads, new token).  A page of 32 tokens comes in once by TMA (slabs of 64 columns,
// 128-byte swizzle) and serves as keys and as values of all N heads:
//   scores   S [heads, tokens] = Q C^T      Q the heads' queries, resident in tensor memory; C the page as it lies (K-major)
//   values   O^T [latent, N] += C^T P^T     C^T the same page read MN-major, P the probabilities (K-major): transposed, so that
//                                           the latent's columns and not the few heads are the 128-row side
// so that every product reads the page's shared memory at most once.  Warp 0 loads; one thread of warp 1 issues S of the next
// page ahead of O^T of this one; warp 4 holds a head per thread (lanes past N heads compute on whatever tensor memory holds
// there, and nobody reads it).  A head's reference for its exponentials is only raised when its maximum has grown by more than
// 2^8 since it was last set (see attn_prefill.cu); warps 4-7 then rescale O^T in tensor memory.
// The splits of a token are a cluster: each leaves its unnormalised sums in shared memory, and each adds up a share of the
// heads from all of them.  NS: slabs of a row; VS: slabs of its latent.
constexpr int kLatMaxSplits = 8;
constexpr float kLatRescaleStep = 8.f;
enum { LAT_STEADY = 0, LAT_RAISE = 1, LAT_ABORT = 2 };

struct LatentMmaParams {
  NkbLatentArgs a;
  const __nv_bfloat16* q;
  const int *block_table, *q_start, *q_lens, *context_lens;
  __nv_bfloat16* out;
  int* status;
  int batch, max_blocks, num_splits;
  float scale_log2;
};

template <int NS, int VS, int N>
struct LatentSmem {
  static constexpr int kSlab = kLatPage * 128, kStage = NS * kSlab;
  static constexpr int kStages = NS >= 5 ? 5 : 8;
  static constexpr int kProb = N * 128;
  static constexpr int kP = kStages * kStage;                      // two buffers
  static constexpr int kEnd = kP + 2 * kProb;
  static constexpr int kOLd = VS * 64 + 8;                         // of the sums that splits exchange, in the ring's place
  static constexpr int kTiles = (VS + 1) / 2;                      // 128-row tiles of O^T
  // tensor memory: two buffers of S, the queries (two elements a column), O^T
  static constexpr int kSCol = 0, kQCol = 2 * kLatPage, kOCol = kQCol + NS * 32;
  static constexpr int kUsed = kOCol + kTiles * N;
  static constexpr int kCols = kUsed <= 128 ? 128 : (kUsed <= 256 ? 256 : 512);
  static_assert(N * kOLd * 4 <= kP && kUsed <= 512, "what splits exchange fits in the ring");
};

__device__ __forceinline__ float ld_cluster(uint32_t addr) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
  return v;
}
__device__ __forceinline__ float4 ld_cluster4(uint32_t addr) {
  float4 v;
  asm volatile("ld.shared::cluster.v4.f32 {%0, %1, %2, %3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(addr) : "memory");
  return v;
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
template <int N>
__device__ __forceinline__ void tmem_ld_cols(uint32_t addr, uint32_t (&r)[N]) {
  if constexpr (N == 32) tmem_ld_32x32(addr, r);
  else tmem_ld_32x16(addr, r);
}
template <int N>
__device__ __forceinline__ void tmem_st_cols(uint32_t addr, const uint32_t (&r)[N]) {
  if constexpr (N == 32) tmem_st_32x32(addr, r);
  else tmem_st_32x16(addr, r);
}
template <int NS, int VS, int N>
__global__ void __launch_bounds__(256, 1)
latent_attn_kernel(const __grid_constant__ CUtensorMap tmC, const __grid_constant__ LatentMmaParams p) {
  using L = LatentSmem<NS, VS, N>;
  constexpr int VC = VS * 64;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* p_s = smem + L::kP;
  __shared__ uint64_t q_ready, kv_full[L::kStages], kv_empty[L::kStages], s_full[2], s_empty[2], p_full[2], p_empty[2];
  __shared__ uint32_t tmem_s;
  __shared__ __align__(16) float raise_s[N], m_s[N], l_s[N], sc_s[kLatMaxSplits][N];
  __shared__ int abort_s, state_s[2];
  const int warp = warp_idx_uniform(), lane = threadIdx.x & 31;
  const int split = blockIdx.x, head0 = blockIdx.y * N, t = blockIdx.z;
  const int nh = min(N, p.a.heads - head0);
  if (threadIdx.x == 0) {
    tma_prefetch_desc(&tmC);
    mbar_init(&q_ready, 1);
    for (int s = 0; s < L::kStages; ++s) {
      mbar_init(&kv_full[s], 1);
      mbar_init(&kv_empty[s], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&s_empty[i], 1);
      mbar_init(&p_full[i], 4);
      mbar_init(&p_empty[i], 1);
    }
    abort_s = 0;
    mbar_fence_init();
    fence_proxy_async();
  }
  griddep_wait();
  // between the two: neither the kernel before this one nor the one after it can wait for tensor memory that this one holds
  if (warp == 1) {
    tmem_alloc(&tmem_s, L::kCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  griddep_launch();
  const uint32_t tmem = __shfl_sync(0xffffffffu, tmem_s, 0);
  volatile int* abort_flag = &abort_s;
  int b = -1, pos = -1;
  if (!p.q_lens) {
    b = t;
    pos = p.context_lens[t] - 1;
  } else {
    for (int i = 0; i < p.batch; ++i) {
      const int r = t - p.q_start[i];
      if (r >= 0 && r < p.q_lens[i]) {
        b = i;
        pos = p.context_lens[i] - p.q_lens[i] + r;
      }
    }
  }
  __nv_bfloat16* out = p.out + t * p.a.o_token + head0 * p.a.o_head;
  if (pos < 0) {
    if (split == 0)
      for (int i = threadIdx.x; i < nh * p.a.rank; i += 256)
        out[(i / p.a.rank) * p.a.o_head + i % p.a.rank] = __float2bfloat16(0.f);
    if (warp == 1) tmem_dealloc(tmem, L::kCols);
    return;
  }
  const int lo = nkb_first_visible(pos, p.a.window, 0);
  const int page_lo = lo / kLatPage, npages = pos / kLatPage + 1 - page_lo;
  const int per_split = (npages + p.num_splits - 1) / p.num_splits;
  const int p0 = page_lo + split * per_split, n = max(0, min(page_lo + npages, p0 + per_split) - p0);

  if (warp == 0) {
    // ---------------------------------------------------------------- loads
    const int* table = p.block_table + (long long)b * p.max_blocks;
    int next = n > 0 ? table[p0] : 0;
    for (int i = 0; i < n; ++i) {
      const int st = i % L::kStages, blk = next;
      if (i + 1 < n) next = table[p0 + i + 1];
      const bool ok = mbar_wait(&kv_empty[st], (uint32_t(i / L::kStages) & 1u) ^ 1u, abort_flag, p.status, ERR_WAIT_SMEM_EMPTY);
      if (!__all_sync(0xffffffffu, ok)) break;
      if (lane == 0) {
        uint8_t* dst = smem + st * L::kStage;
        mbar_expect_tx(&kv_full[st], L::kStage);
#pragma unroll
        for (int s = 0; s < NS; ++s) tma_load_3d(dst + s * L::kSlab, &tmC, &kv_full[st], s * 64, 0, blk);
      }
      __syncwarp();
    }
  } else if (warp == 1) {
    // ---------------------------------------------------------------- products
    constexpr uint32_t idesc_s = make_idesc_bf16(128, kLatPage, 0, 0), idesc_o = make_idesc_bf16(128, N, 1, 0);
    const uint64_t hk = uint64_t(uint32_t(make_smem_desc_sw128(0, 0, 1024) >> 32)) << 32;      // SBO, version, swizzle
    const uint32_t c_lo = uint32_t(make_smem_desc_sw128(smem_u32(smem), 0, 1024));
    const uint32_t p_lo = uint32_t(make_smem_desc_sw128(smem_u32(p_s), 0, 1024));
    constexpr uint32_t lbo = (uint32_t(L::kSlab) >> 4) << 16;                                    // next 64 columns of C^T
    if (n > 0 && elect_one()) {
      bool ok = mbar_wait(&q_ready, 0, abort_flag, p.status, ERR_WAIT_SOFTMAX);
      const auto scores = [&](int i) {
        const int st = i % L::kStages, buf = i & 1;
        ok = ok && mbar_wait(&kv_full[st], uint32_t(i / L::kStages) & 1u, abort_flag, p.status, ERR_WAIT_SMEM_FULL);
        ok = ok && mbar_wait(&s_empty[buf], (uint32_t(i / 2) & 1u) ^ 1u, abort_flag, p.status, ERR_WAIT_TMEM_EMPTY);
        if (!ok) return;
        tc_fence_after();
#pragma unroll
        for (int k = 0; k < 4 * NS; ++k)
          umma_f16_ts(tmem + L::kSCol + buf * kLatPage, tmem + L::kQCol + k * 8,
                      hk | (c_lo + uint32_t((st * L::kStage + (k >> 2) * L::kSlab) >> 4) + (k & 3) * 2), idesc_s, k > 0 ? 1u : 0u);
        umma_commit(&s_full[buf]);
      };
      scores(0);
      for (int i = 0; i < n && ok; ++i) {
        if (i + 1 < n) scores(i + 1);
        const int st = i % L::kStages, buf = i & 1;
        ok = ok && mbar_wait(&p_full[buf], uint32_t(i / 2) & 1u, abort_flag, p.status, ERR_WAIT_SOFTMAX);
        if (!ok) break;
        tc_fence_after();
#pragma unroll
        for (int m = 0; m < L::kTiles; ++m) {
#pragma unroll
          for (int k = 0; k < 2; ++k)              // sixteen tokens a step
            umma_f16(tmem + L::kOCol + m * N, hk | ((c_lo + uint32_t((st * L::kStage + 2 * m * L::kSlab) >> 4) + k * 128) | lbo),
                     hk | (p_lo + uint32_t(buf * L::kProb >> 4) + k * 2), idesc_o, i > 0 || k > 0 ? 1u : 0u);
        }
        umma_commit(&p_empty[buf]);
        umma_commit(&kv_empty[st]);
      }
    }
    __syncwarp();
  } else if (warp >= 4) {
    // ---------------------------------------------------------------- softmax
    const int quad = warp & 3, tok = quad * 32 + lane;
    const uint32_t lanes = uint32_t(quad * 32) << 16;
    const bool holds = quad == 0;                   // the warp with the heads
    if (holds && n > 0) {
      // queries of head `lane` -> tensor memory, half a row's slabs at a time so that their loads are in flight together
      const uint4* q = reinterpret_cast<const uint4*>(p.q + t * p.a.q_token + (head0 + lane) * p.a.q_head);
      constexpr int kHalf = (NS + 1) / 2;
#pragma unroll
      for (int s0 = 0; s0 < NS; s0 += kHalf) {
        uint32_t r[kHalf][32];
#pragma unroll
        for (int s = 0; s < kHalf; ++s)
#pragma unroll
          for (int c = 0; c < 8; ++c) {
            const uint4 w = s0 + s < NS && lane < nh ? q[(s0 + s) * 8 + c] : make_uint4(0u, 0u, 0u, 0u);
            r[s][4 * c] = w.x; r[s][4 * c + 1] = w.y; r[s][4 * c + 2] = w.z; r[s][4 * c + 3] = w.w;
          }
#pragma unroll
        for (int s = 0; s < kHalf; ++s)
          if (s0 + s < NS) tmem_st_32x32(tmem + L::kQCol + (s0 + s) * 32, r[s]);
      }
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&q_ready);
    }
    float l = 0.f, m = -INFINITY;                   // of head `lane`
    bool alive = true;
    for (int i = 0; i < n; ++i) {
      const int buf = i & 1;
      float x[kLatPage], mx = -INFINITY;
      bool grow = false;
      if (holds) {
        alive = alive && mbar_wait(&s_full[buf], uint32_t(i / 2) & 1u, abort_flag, p.status, ERR_WAIT_TMEM_FULL);
        alive = __all_sync(0xffffffffu, alive);
        int state = LAT_ABORT;
        if (alive) {
          uint32_t r[kLatPage];
          tc_fence_after();
          tmem_ld_32x32(tmem + L::kSCol + buf * kLatPage, r);
          tmem_ld_wait();
          tc_fence_before();
          __syncwarp();
          if (lane == 0) mbar_arrive(&s_empty[buf]);
          const int first = lo - (p0 + i) * kLatPage, last = pos - (p0 + i) * kLatPage;
#pragma unroll
          for (int j = 0; j < kLatPage; ++j) x[j] = __uint_as_float(r[j]) * p.scale_log2;
          if (first > 0 || last < kLatPage - 1) {   // the same for all lanes
#pragma unroll
            for (int j = 0; j < kLatPage; ++j)
              if (j < first || j > last) x[j] = -INFINITY;
          }
          float m4[4] = {x[0], x[1], x[2], x[3]};
#pragma unroll
          for (int j = 4; j < kLatPage; ++j) m4[j & 3] = fmaxf(m4[j & 3], x[j]);
          mx = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3]));      // finite: every page holds a visible token
          grow = lane < nh && (mx > m + kLatRescaleStep || m == -INFINITY);
          if (i == 0) {                             // nothing to rescale
            if (grow) m = mx;
            grow = false;
          }
          state = __any_sync(0xffffffffu, grow) ? LAT_RAISE : LAT_STEADY;
        }
        if (lane == 0) state_s[buf] = state;
      }
      asm volatile("bar.sync 1, 128;" ::: "memory");
      const int state = state_s[buf];
      if (state == LAT_ABORT) break;
      if (state == LAT_RAISE) {
        if (holds) {
          const float alpha = grow ? ex2(m - mx) : 1.f;
          if (lane < N) raise_s[lane] = alpha;
          if (grow) m = mx;
          l *= alpha;
        }
        asm volatile("bar.sync 1, 128;" ::: "memory");
        // O^T holds all of the page before this one
        alive = alive && mbar_wait(&p_empty[buf ^ 1], uint32_t((i - 1) / 2) & 1u, abort_flag, p.status, ERR_WAIT_TMEM_FULL);
        alive = __all_sync(0xffffffffu, alive);
        tc_fence_after();
#pragma unroll 1
        for (int tile = 0; tile < L::kTiles; ++tile) {
          uint32_t o[N];
          tmem_ld_cols<N>(tmem + lanes + L::kOCol + tile * N, o);
          tmem_ld_wait();
#pragma unroll
          for (int h = 0; h < N; ++h) o[h] = __float_as_uint(__uint_as_float(o[h]) * raise_s[h]);
          tmem_st_cols<N>(tmem + lanes + L::kOCol + tile * N, o);
        }
        tmem_st_wait();
      }
      if (holds) {
        const float base = m == -INFINITY ? 0.f : m;             // lanes without a head
        float l4[4] = {0.f, 0.f, 0.f, 0.f};
        uint32_t pk[kLatPage / 2];
#pragma unroll
        for (int j = 0; j < kLatPage; j += 2) {
          const float e0 = ex2(x[j] - base), e1 = ex2(x[j + 1] - base);
          l4[j & 2] += e0;
          l4[(j & 2) + 1] += e1;
          pk[j / 2] = pack_bf16x2(e0, e1);
        }
        l += (l4[0] + l4[1]) + (l4[2] + l4[3]);
        if (i >= 2) {                               // the buffer's probabilities have been multiplied
          alive = alive && mbar_wait(&p_empty[buf], uint32_t(i / 2 - 1) & 1u, abort_flag, p.status, ERR_WAIT_TMEM_FULL);
          alive = __all_sync(0xffffffffu, alive);
        }
        if (lane < N) {
          uint8_t* dst = p_s + buf * L::kProb + lane * 128;
#pragma unroll
          for (int c = 0; c < 4; ++c)
            *reinterpret_cast<uint4*>(dst + ((c ^ (lane & 7)) << 4)) = make_uint4(pk[4 * c], pk[4 * c + 1], pk[4 * c + 2], pk[4 * c + 3]);
        }
        fence_proxy_async();
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[buf]);
    }
    // ---- all pages: O^T out of tensor memory
    if (n > 0) {
      alive = alive && mbar_wait(&p_empty[(n - 1) & 1], uint32_t((n - 1) / 2) & 1u, abort_flag, p.status, ERR_WAIT_TMEM_FULL);
      alive = __all_sync(0xffffffffu, alive);
      tc_fence_after();
    }
    if (holds && lane < N) {
      m_s[lane] = lane < nh ? m : -INFINITY;
      l_s[lane] = l;
    }
    float* o_s = reinterpret_cast<float*>(smem);                      // every page has been consumed
#pragma unroll 1
    for (int tile = 0; tile < L::kTiles; ++tile) {
      uint32_t o[N];
      if (n > 0) {
        tmem_ld_cols<N>(tmem + lanes + L::kOCol + tile * N, o);
        tmem_ld_wait();
      } else {
#pragma unroll
        for (int h = 0; h < N; ++h) o[h] = 0u;
      }
      const int c = tile * 128 + tok;
      if (c < VC) {
#pragma unroll
        for (int h = 0; h < N; ++h) o_s[h * L::kOLd + c] = __uint_as_float(o[h]);
      }
    }
    tc_fence_before();
  }
  if (*abort_flag) {
    for (int i = 0; i < 200; ++i) __nanosleep(1000);
  }
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, L::kCols);
  }
  const float* o_s = reinterpret_cast<const float*>(smem);
  if (p.num_splits > 1) cluster_sync_all();
  // this CTA's heads: r0 .. r0 + per - 1
  const int splits = p.num_splits, per = N / splits, r0 = split * per;
  if (int(threadIdx.x) < per) {
    const int r = r0 + threadIdx.x;
    const float sk = r < nh && p.a.sinks ? p.a.sinks[head0 + r] * 1.4426950408889634f : -INFINITY;
    float ms[kLatMaxSplits], ls[kLatMaxSplits], mf = sk, den = 0.f;
#pragma unroll
    for (int s = 0; s < kLatMaxSplits; ++s)
      if (s < splits) {
        ms[s] = ld_cluster(map_to_cta(&m_s[r], s));
        ls[s] = ld_cluster(map_to_cta(&l_s[r], s));
      }
#pragma unroll
    for (int s = 0; s < kLatMaxSplits; ++s)
      if (s < splits) mf = fmaxf(mf, ms[s]);
#pragma unroll
    for (int s = 0; s < kLatMaxSplits; ++s)
      if (s < splits) {
        ms[s] = ms[s] > -INFINITY ? exp2f(ms[s] - mf) : 0.f;
        den += ms[s] * ls[s];
      }
    if (sk > -INFINITY) den += exp2f(sk - mf);
#pragma unroll
    for (int s = 0; s < kLatMaxSplits; ++s)
      if (s < splits) sc_s[s][threadIdx.x] = ms[s] / den;
  }
  __syncthreads();
  uint32_t peer[kLatMaxSplits];
#pragma unroll
  for (int s = 0; s < kLatMaxSplits; ++s) peer[s] = s < splits ? map_to_cta(o_s, s) : 0u;
#pragma unroll 2
  for (int i = threadIdx.x * 4; i < per * VC; i += 1024) {
    const int r = i / VC, c = i % VC;
    float4 x[kLatMaxSplits];
#pragma unroll
    for (int s = 0; s < kLatMaxSplits; ++s)
      if (s < splits) x[s] = ld_cluster4(peer[s] + ((r0 + r) * L::kOLd + c) * 4);
    float v[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int s = 0; s < kLatMaxSplits; ++s)
      if (s < splits) {
        const float sc = sc_s[s][r];
        v[0] = fmaf(sc, x[s].x, v[0]); v[1] = fmaf(sc, x[s].y, v[1]);
        v[2] = fmaf(sc, x[s].z, v[2]); v[3] = fmaf(sc, x[s].w, v[3]);
      }
    if (r0 + r >= nh) continue;
    __nv_bfloat16* dst = out + (r0 + r) * p.a.o_head + c;
    if (c + 3 < p.a.rank && ((p.a.o_head | p.a.o_token) & 3) == 0) {
      *reinterpret_cast<uint2*>(dst) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (c + e < p.a.rank) dst[e] = __float2bfloat16(v[e]);
    }
  }
  if (p.num_splits > 1) cluster_sync_all();          // no CTA leaves while its sums are read
}

template <int NS, int VS, int N>
static int launch_latent(const CUtensorMap& tc, const LatentMmaParams& p, int tokens, cudaStream_t s) {
  using L = LatentSmem<NS, VS, N>;
  constexpr int smem = L::kEnd + 1024;
  static_assert(smem + 3072 <= 232448, "shared memory of a CTA");
  static bool attr_set[64] = {false};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -1;
  if (!attr_set[dev]) {
    cudaError_t e = cudaFuncSetAttribute(latent_attn_kernel<NS, VS, N>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return int(e);
    attr_set[dev] = true;
  }
  const dim3 grid(p.num_splits, (p.a.heads + N - 1) / N, tokens);
  return launch_pdl_cluster(latent_attn_kernel<NS, VS, N>, grid, dim3(256), size_t(smem), s, p.num_splits, tc, p);
}
template <int NS, int VS>
static int launch_latent_heads(const CUtensorMap& tc, const LatentMmaParams& p, int tokens, cudaStream_t s) {
  return p.a.heads <= 16 ? launch_latent<NS, VS, 16>(tc, p, tokens, s) : launch_latent<NS, VS, 32>(tc, p, tokens, s);
}

// Slabs of a row and of its latent that the kernel is built for; 0 when it does not take the sizes.
static int latent_shape(const NkbLatentArgs& a, int* vs) {
  static const int shapes[][2] = {{2, 1}, {3, 2}, {5, 4}, {9, 8}};
  for (const auto& s : shapes)
    if (a.rank <= s[1] * 64 && a.rank + a.rot <= s[0] * 64) {
      *vs = s[1];
      return s[0];
    }
  return 0;
}

static bool latent_ok(const NkbLatentArgs& a) {
  return a.heads >= 1 && a.dim >= 1 && a.rot >= 2 && (a.rot & 1) == 0 && a.rank >= 1 && a.q_rank >= 1 && a.row >= a.rank + a.rot;
}
static bool al16(const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; }

}  // namespace nkb

using namespace nkb;

extern "C" int nkb_latent_append(const NkbLatentArgs* a, const NkbProj* q, const NkbProj* kv, const float* q_norm,
                                 const float* kv_norm, const float* cos_sin, int max_pos, const int* positions,
                                 const int* slots, void* q_out, void* cache, int bf16, int tokens, int block_size,
                                 void* stream) {
  if (tokens <= 0) return 0;
  if (!latent_ok(*a) || block_size != kLatPage || max_pos < 1) return -2;
  LatentAppendParams p{*q, *kv, *a, q_norm, kv_norm, cos_sin, positions, slots, q_out, cache, max_pos};
  const size_t smem = size_t((a->q_rank + 3) / 4 * 4 + a->rank) * sizeof(float);
  if (smem > 48 * 1024 - 128) return -2;
  const bool vec = ((a->q_rank | a->rank | a->rot | a->row) & 3) == 0 && proj_vec4_ok(*q) && proj_vec4_ok(*kv) && al16(q_out) &&
                   al16(cache);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  using bf = __nv_bfloat16;
  const dim3 grid(tokens), block(256);
  if (bf16 && q->bf16 && kv->bf16 && a->q_rank <= 256 * kAppendQ && a->rank <= 256 * kAppendK && a->row - a->rank <= 256 &&
      ((a->q_rank | a->rank | a->rot | a->row) & 7) == 0 && ((q->ld | kv->ld) & 7) == 0 && al16(q->ptr) && al16(kv->ptr) &&
      al16(q_out) && al16(cache) && al16(q_norm) && al16(kv_norm) && al16(cos_sin))
    return launch_pdl(latent_append8_kernel, dim3((tokens + 7) / 8), block, 0, s, p, tokens);
  if (vec)
    return bf16 ? launch_pdl(latent_append_kernel<4, bf>, grid, block, smem, s, p)
                : launch_pdl(latent_append_kernel<4, float>, grid, block, smem, s, p);
  return bf16 ? launch_pdl(latent_append_kernel<1, bf>, grid, block, smem, s, p)
              : launch_pdl(latent_append_kernel<1, float>, grid, block, smem, s, p);
}

extern "C" int nkb_latent_queries(const NkbLatentArgs* a, const NkbProj* q, const float* cos_sin, int max_pos,
                                  const int* positions, void* plain, long long plain_token, long long plain_head, int plain_pad,
                                  void* rotated, long long rot_token, long long rot_head, int rot_pad, int bf16, int tokens,
                                  void* stream) {
  if (tokens <= 0) return 0;
  if (!latent_ok(*a) || plain_pad < a->dim || rot_pad < a->rot || max_pos < 1) return -2;
  LatentQueryParams p{*q, *a, cos_sin, positions, plain, rotated, plain_token, plain_head, rot_token, rot_head,
                      (long long)tokens * a->heads, plain_pad, rot_pad, max_pos};
  if (p.rows > 0x7fffffffll / 32) return -2;
  const long long strides = plain_token | plain_head | rot_token | rot_head;
  const bool vec = ((a->dim | a->rot | plain_pad | rot_pad) & 3) == 0 && (strides & 3) == 0 && proj_vec4_ok(*q) &&
                   (reinterpret_cast<uintptr_t>(plain) & (bf16 ? 7 : 15)) == 0 &&
                   (reinterpret_cast<uintptr_t>(rotated) & (bf16 ? 7 : 15)) == 0;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  using bf = __nv_bfloat16;
  const dim3 grid(unsigned((p.rows + 7) / 8)), block(256);
  if (bf16 && q->bf16 && ((a->dim | a->rot | plain_pad | rot_pad) & 7) == 0 && (strides & 7) == 0 && (q->ld & 7) == 0 &&
      al16(q->ptr) && al16(plain) && al16(rotated) && al16(cos_sin))
    return launch_pdl(latent_query8_kernel, dim3(tokens), block, 0, s, p);
  if (vec)
    return bf16 ? launch_pdl(latent_query_kernel<4, bf>, grid, block, 0, s, p)
                : launch_pdl(latent_query_kernel<4, float>, grid, block, 0, s, p);
  return bf16 ? launch_pdl(latent_query_kernel<1, bf>, grid, block, 0, s, p)
              : launch_pdl(latent_query_kernel<1, float>, grid, block, 0, s, p);
}

extern "C" int nkb_latent_gather(const void* cache, const int* pages, int n_pages, int row, int rank, int rot, int rot_ld,
                                 void* c_out, void* r_out, int bf16, int block_size, void* stream) {
  if (n_pages <= 0) return 0;
  if (block_size != kLatPage || rank < 1 || rot < 1 || row < rank + rot || rot_ld < rot || !al16(cache) || !al16(c_out) ||
      !al16(r_out) || (row * (bf16 ? 2 : 4)) % 16)
    return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  using bf = __nv_bfloat16;
  if (bf16)
    return launch_pdl(latent_gather_kernel<bf>, dim3(n_pages), dim3(256), 0, s, (const bf*)cache, pages, row, rank, rot, rot_ld,
                      (bf*)c_out, (bf*)r_out);
  return launch_pdl(latent_gather_kernel<float>, dim3(n_pages), dim3(256), 0, s, (const float*)cache, pages, row, rank, rot,
                    rot_ld, (float*)c_out, (float*)r_out);
}

// Attention of new tokens, already in the cache, over the visible cached rows; queries and results as latents, bf16.  q_lens null:
// token t belongs to sequence t.  num_splits is rounded down to 1, 2, 4 or 8.  Returns -5 for sizes it does not take.
extern "C" int nkb_latent_attn(const NkbLatentArgs* a, const void* q, const void* cache, const int* block_table,
                               const int* q_start, const int* q_lens, const int* context_lens, void* out, int batch,
                               int tokens, int block_size, int num_blocks, int max_blocks_per_seq, int num_splits,
                               void* stream) {
  if (batch <= 0 || tokens <= 0) return 0;
  int vs = 0;
  const int ns = latent_shape(*a, &vs);
  if (!ns || a->row != ns * 64) return -5;
  if (!latent_ok(*a) || block_size != kLatPage || tokens > 65535 || (!q_lens && tokens != batch)) return -2;
  if (!al16(q) || ((a->q_token | a->q_head) & 7) || (reinterpret_cast<uintptr_t>(out) & 7)) return -2;
  if (!status_word() && nkb_init() != 0) return -1;
  LatentMmaParams p{};
  p.a = *a;
  p.q = reinterpret_cast<const __nv_bfloat16*>(q);
  const int splits = num_splits >= 8 ? 8 : num_splits >= 4 ? 4 : num_splits >= 2 ? 2 : 1;
  p.block_table = block_table; p.q_start = q_start; p.q_lens = q_lens; p.context_lens = context_lens;
  p.out = reinterpret_cast<__nv_bfloat16*>(out);
  p.status = status_word();
  p.batch = batch; p.max_blocks = max_blocks_per_seq; p.num_splits = splits;
  p.scale_log2 = a->scale * 1.4426950408889634f;
  CUtensorMap tc;
  const uint64_t dims[3] = {uint64_t(a->row), uint64_t(kLatPage), uint64_t(num_blocks)};
  const uint64_t strides[2] = {uint64_t(a->row) * 2, uint64_t(a->row) * kLatPage * 2};
  const uint32_t box[3] = {64, uint32_t(kLatPage), 1};
  if (encode_tmap_bf16(&tc, cache, 3, dims, strides, box)) return -4;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  switch (ns) {
    case 2: return launch_latent_heads<2, 1>(tc, p, tokens, s);
    case 3: return launch_latent_heads<3, 2>(tc, p, tokens, s);
    case 5: return launch_latent_heads<5, 4>(tc, p, tokens, s);
    default: return launch_latent_heads<9, 8>(tc, p, tokens, s);
  }
}
