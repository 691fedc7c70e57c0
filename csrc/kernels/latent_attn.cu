// Latent attention (latent_attn.h) over a paged cache of latents:
//   append    the two down projections of a token: the query latent RMS-normed, the key / value latent RMS-normed and the
//             shared key part rotated (pairs 2i, 2i + 1) into the token's cache row
//   queries   the up-projected queries split into their unrotated and rotated parts, the latter rotated
//   gather    cached rows of whole pages as two matrices, the operands of the up projections of keys and values
//   attention any new tokens against the cached rows themselves, bf16: see latent_mma_kernel
#include "common.cuh"
#include "mma_frag.cuh"
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
// One CTA of four warps per (split of the visible pages, 16 MT heads, new token).  A page's rows come in once by TMA (slabs of
// 64 columns, 128-byte swizzle) and serve as keys and as values of all heads:
//   scores   every warp contracts a quarter of the row's columns; the queries of its quarter stay in registers as MMA
//            fragments.  The four partial products meet in shared memory.
//   softmax  128 / (16 MT) threads per head sum the partials, mask, and keep the running maximum and denominator
//   values   every warp multiplies the probabilities with a quarter of the latent's columns
// Two block barriers per page.  Splits are merged by the CTA that arrives last, as in attn_decode.cu.
// NS: slabs of a row; VS: slabs of its latent.
constexpr int kLatCounters = 16384;   // arrival counters in front of the split partials

struct LatentMmaParams {
  NkbLatentArgs a;
  const __nv_bfloat16* q;
  const int *block_table, *q_start, *q_lens, *context_lens;
  __nv_bfloat16* out;
  float* scratch;
  unsigned int* counters;
  int* status;
  int batch, max_blocks, num_splits;
  float scale_log2;
};

template <int NS>
struct LatentStages {
  static constexpr int value = NS >= 8 ? 2 : 3;
};

template <int NS, int VS, int MT>
struct LatentSmem {
  static constexpr int kSlab = kLatPage * 128, kStage = NS * kSlab, kStages = LatentStages<NS>::value;
  static constexpr int kRows = 16 * MT, kSLd = 36, kPLd = 40;      // leading dimensions of scores (fp32) and probabilities
  static constexpr int kScores = kStages * kStage;
  static constexpr int kProbs = kScores + 4 * kRows * kSLd * 4;
  static constexpr int kEnd = kProbs + kRows * kPLd * 2;
};

template <int NS, int VS, int MT>
__global__ void __launch_bounds__(128, 2)
latent_mma_kernel(const __grid_constant__ CUtensorMap tmC, const __grid_constant__ LatentMmaParams p) {
  using L = LatentSmem<NS, VS, MT>;
  constexpr int kRows = L::kRows, VC = VS * 64, TPR = 128 / kRows, PER = kLatPage / TPR;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  float* s_s = reinterpret_cast<float*>(smem + L::kScores);                       // [4][kRows][kSLd]
  __nv_bfloat16* p_s = reinterpret_cast<__nv_bfloat16*>(smem + L::kProbs);        // [kRows][kPLd]
  __shared__ uint64_t bars[L::kStages];
  __shared__ float al_s[kRows], m_s[kRows], l_s[kRows];
  __shared__ int abort_flag, is_last;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3;
  const int split = blockIdx.x, head0 = blockIdx.y * kRows, t = blockIdx.z;
  const int nh = min(kRows, p.a.heads - head0);
  if (threadIdx.x == 0) {
    for (int s = 0; s < L::kStages; ++s) mbar_init(&bars[s], 1);
    abort_flag = 0;
    mbar_fence_init();
    fence_proxy_async();
    tma_prefetch_desc(&tmC);
  }
  __syncthreads();
  griddep_wait();
  griddep_launch();
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
      for (int i = threadIdx.x; i < nh * p.a.rank; i += 128)
        out[(i / p.a.rank) * p.a.o_head + i % p.a.rank] = __float2bfloat16(0.f);
    return;
  }
  const int lo = nkb_first_visible(pos, p.a.window, 0);
  const int page_lo = lo / kLatPage, npages = pos / kLatPage + 1 - page_lo;
  const int per_split = (npages + p.num_splits - 1) / p.num_splits;
  const int p0 = page_lo + split * per_split, n = max(0, min(page_lo + npages, p0 + per_split) - p0);
  const int* table = p.block_table + (long long)b * p.max_blocks;
  auto issue = [&](int i) {
    const int st = i % L::kStages, blk = table[p0 + i];
    mbar_expect_tx(&bars[st], L::kStage);
#pragma unroll
    for (int s = 0; s < NS; ++s) tma_load_3d(smem + st * L::kStage + s * L::kSlab, &tmC, &bars[st], s * 64, 0, blk);
  };
  if (threadIdx.x == 0)
    for (int i = 0; i < L::kStages && i < n; ++i) issue(i);

  uint32_t qf[MT][NS][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt) {
    const int r0 = mt * 16 + g, r1 = r0 + 8;
    const __nv_bfloat16* q0 = p.q + t * p.a.q_token + (head0 + r0) * p.a.q_head;
    const __nv_bfloat16* q1 = q0 + 8 * p.a.q_head;
#pragma unroll
    for (int k = 0; k < NS; ++k) {
      const int c = (warp * NS + k) * 16 + 2 * tq;
      qf[mt][k][0] = r0 < nh ? *reinterpret_cast<const uint32_t*>(q0 + c) : 0u;
      qf[mt][k][1] = r1 < nh ? *reinterpret_cast<const uint32_t*>(q1 + c) : 0u;
      qf[mt][k][2] = r0 < nh ? *reinterpret_cast<const uint32_t*>(q0 + c + 8) : 0u;
      qf[mt][k][3] = r1 < nh ? *reinterpret_cast<const uint32_t*>(q1 + c + 8) : 0u;
    }
  }
  float o[MT][2 * VS][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int i = 0; i < 2 * VS; ++i) o[mt][i][0] = o[mt][i][1] = o[mt][i][2] = o[mt][i][3] = 0.f;
  const int row = threadIdx.x / TPR, sub = threadIdx.x % TPR;
  float m = -INFINITY, l = 0.f;

  for (int i = 0; i < n; ++i) {
    const int st = i % L::kStages;
    const bool ok = mbar_wait(&bars[st], uint32_t(i / L::kStages) & 1u, &abort_flag, p.status, ERR_WAIT_SMEM_FULL);
    const uint32_t base = smem_u32(smem + st * L::kStage);
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      float s[MT][2][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) s[mt][nt][0] = s[mt][nt][1] = s[mt][nt][2] = s[mt][nt][3] = 0.f;
#pragma unroll
      for (int k = 0; k < NS; ++k) {
        // two groups of eight tokens by sixteen columns
        const int tok = half * 16 + (lane >> 4) * 8 + (lane & 7), ch = 2 * (warp * NS + k) + ((lane >> 3) & 1);
        uint32_t b0, b1, b2, b3;
        ldsm_x4(base + (ch >> 3) * L::kSlab + tok * 128 + (((ch & 7) ^ (tok & 7)) << 4), b0, b1, b2, b3);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          mma_16816(s[mt][0], qf[mt][k], b0, b1);
          mma_16816(s[mt][1], qf[mt][k], b2, b3);
        }
      }
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          float* d = s_s + (warp * kRows + mt * 16 + g) * L::kSLd + half * 16 + nt * 8 + 2 * tq;
          *reinterpret_cast<float2*>(d) = make_float2(s[mt][nt][0], s[mt][nt][1]);
          *reinterpret_cast<float2*>(d + 8 * L::kSLd) = make_float2(s[mt][nt][2], s[mt][nt][3]);
        }
    }
    if (!__syncthreads_and(ok)) break;
    // every warp is done with the page before this one: its stage is free
    if (threadIdx.x == 0 && i > 0 && i - 1 + L::kStages < n) issue(i - 1 + L::kStages);
    float x[PER], mx = -INFINITY;
    {
      const float* sp = s_s + row * L::kSLd + sub * PER;
#pragma unroll
      for (int j = 0; j < PER; j += 4) {
        float4 a = *reinterpret_cast<const float4*>(sp + j);
#pragma unroll
        for (int w = 1; w < 4; ++w) {
          const float4 c = *reinterpret_cast<const float4*>(sp + w * kRows * L::kSLd + j);
          a.x += c.x; a.y += c.y; a.z += c.z; a.w += c.w;
        }
        x[j] = a.x; x[j + 1] = a.y; x[j + 2] = a.z; x[j + 3] = a.w;
      }
      const int tok0 = (p0 + i) * kLatPage + sub * PER;
#pragma unroll
      for (int j = 0; j < PER; ++j) {
        x[j] = tok0 + j >= lo && tok0 + j <= pos ? x[j] * p.scale_log2 : -INFINITY;
        mx = fmaxf(mx, x[j]);
      }
    }
#pragma unroll
    for (int w = 1; w < TPR; w <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, w));
    const float mn = fmaxf(m, mx), alpha = exp2f(m - mn);      // finite: every page holds a visible token
    m = mn;
    float sum = 0.f;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
      x[j] = exp2f(x[j] - mn);
      sum += x[j];
    }
    l = l * alpha + sum;                                       // this thread's share of the denominator
    __nv_bfloat16* pd = p_s + row * L::kPLd + sub * PER;
#pragma unroll
    for (int j = 0; j < PER; j += 4)
      *reinterpret_cast<uint2*>(pd + j) = make_uint2(pack_bf16x2(x[j], x[j + 1]), pack_bf16x2(x[j + 2], x[j + 3]));
    if (sub == 0) al_s[row] = alpha;
    __syncthreads();
    uint32_t pa[MT][2][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      const float a0 = al_s[mt * 16 + g], a1 = al_s[mt * 16 + g + 8];
#pragma unroll
      for (int u = 0; u < 2 * VS; ++u) {
        o[mt][u][0] *= a0; o[mt][u][1] *= a0;
        o[mt][u][2] *= a1; o[mt][u][3] *= a1;
      }
#pragma unroll
      for (int j = 0; j < 2; ++j)
        ldsm_x4(smem_u32(p_s + (mt * 16 + (lane & 15)) * L::kPLd + 16 * j + (lane >> 4) * 8), pa[mt][j][0], pa[mt][j][1],
                pa[mt][j][2], pa[mt][j][3]);
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int u = 0; u < VS; ++u) {
        const int tok = 16 * j + ((lane >> 3) & 1) * 8 + (lane & 7), ch = 2 * (warp * VS + u) + (lane >> 4);
        uint32_t v0, v1, v2, v3;
        ldsm_x4_t(base + (ch >> 3) * L::kSlab + tok * 128 + (((ch & 7) ^ (tok & 7)) << 4), v0, v1, v2, v3);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          mma_16816(o[mt][2 * u], pa[mt][j], v0, v1);
          mma_16816(o[mt][2 * u + 1], pa[mt][j], v2, v3);
        }
      }
  }
  if (*(volatile int*)&abort_flag) {
    for (int i = 0; i < 200; ++i) __nanosleep(1000);
  }
#pragma unroll
  for (int w = 1; w < TPR; w <<= 1) l += __shfl_xor_sync(0xffffffffu, l, w);
  if (sub == 0) {
    m_s[row] = m;
    l_s[row] = l;
  }
  __syncthreads();
  const auto sink_log2 = [&](int r) { return p.a.sinks ? p.a.sinks[head0 + r] * 1.4426950408889634f : -INFINITY; };
  if (p.num_splits == 1) {
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = mt * 16 + g + 8 * e;
        if (r >= nh) continue;
        const float sk = sink_log2(r), m2 = fmaxf(m_s[r], sk), sc = exp2f(m_s[r] - m2);
        const float inv = sc / (l_s[r] * sc + exp2f(sk - m2));
        __nv_bfloat16* dst = out + r * p.a.o_head;
#pragma unroll
        for (int u = 0; u < 2 * VS; ++u) {
          const int c = warp * VS * 16 + u * 8 + 2 * tq;
          const float v0 = o[mt][u][2 * e] * inv, v1 = o[mt][u][2 * e + 1] * inv;
          if (c + 1 < p.a.rank && ((p.a.o_head | p.a.o_token) & 1) == 0) {
            *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16x2(v0, v1);
          } else {
            if (c < p.a.rank) dst[c] = __float2bfloat16(v0);
            if (c + 1 < p.a.rank) dst[c + 1] = __float2bfloat16(v1);
          }
        }
      }
    return;
  }
  const long long unit = (long long)t * gridDim.y + blockIdx.y;
  constexpr int kPart = kRows * VC + 2 * kRows;
  float* part = p.scratch + (unit * p.num_splits + split) * kPart;
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int u = 0; u < 2 * VS; ++u) {
      float* d = part + (mt * 16 + g) * VC + warp * VS * 16 + u * 8 + 2 * tq;
      *reinterpret_cast<float2*>(d) = make_float2(o[mt][u][0], o[mt][u][1]);
      *reinterpret_cast<float2*>(d + 8 * VC) = make_float2(o[mt][u][2], o[mt][u][3]);
    }
  if (int(threadIdx.x) < kRows) {
    part[kRows * VC + threadIdx.x] = m_s[threadIdx.x];
    part[kRows * VC + kRows + threadIdx.x] = l_s[threadIdx.x];
  }
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
  const float* first = p.scratch + unit * p.num_splits * kPart;
  if (int(threadIdx.x) < kRows) {
    const int r = threadIdx.x;
    float mf = r < nh ? sink_log2(r) : -INFINITY, den = 0.f;
    for (int s = 0; s < p.num_splits; ++s) mf = fmaxf(mf, __ldcg(first + s * kPart + kRows * VC + r));
    if (r < nh && p.a.sinks) den = exp2f(sink_log2(r) - mf);
    for (int s = 0; s < p.num_splits; ++s) {
      const float ms = __ldcg(first + s * kPart + kRows * VC + r);
      if (ms > -INFINITY) den += exp2f(ms - mf) * __ldcg(first + s * kPart + kRows * VC + kRows + r);
    }
    m_s[r] = mf;
    l_s[r] = den;
  }
  __syncthreads();
  for (int i = threadIdx.x * 4; i < nh * VC; i += 512) {
    const int r = i / VC, c = i % VC;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < p.num_splits; ++s) {
      const float* ps = first + s * kPart;
      const float ms = __ldcg(ps + kRows * VC + r), sc = ms > -INFINITY ? exp2f(ms - m_s[r]) : 0.f;
      const float4 x = __ldcg(reinterpret_cast<const float4*>(ps + i));
      acc.x = fmaf(sc, x.x, acc.x); acc.y = fmaf(sc, x.y, acc.y); acc.z = fmaf(sc, x.z, acc.z); acc.w = fmaf(sc, x.w, acc.w);
    }
    const float inv = 1.f / l_s[r], v[4] = {acc.x * inv, acc.y * inv, acc.z * inv, acc.w * inv};
    __nv_bfloat16* dst = out + r * p.a.o_head + c;
#pragma unroll
    for (int e = 0; e < 4; ++e)
      if (c + e < p.a.rank) dst[e] = __float2bfloat16(v[e]);
  }
}

template <int NS, int VS, int MT>
static int launch_latent(const CUtensorMap& tc, const LatentMmaParams& p, int tokens, cudaStream_t s) {
  using L = LatentSmem<NS, VS, MT>;
  constexpr int smem = L::kEnd + 1024;
  static bool attr_set[64] = {false};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -1;
  if (!attr_set[dev]) {
    cudaError_t e = cudaFuncSetAttribute(latent_mma_kernel<NS, VS, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return int(e);
    attr_set[dev] = true;
  }
  const dim3 grid(p.num_splits, (p.a.heads + L::kRows - 1) / L::kRows, tokens);
  return launch_pdl(latent_mma_kernel<NS, VS, MT>, grid, dim3(128), size_t(smem), s, tc, p);
}
template <int NS, int VS>
static int launch_latent_heads(const CUtensorMap& tc, const LatentMmaParams& p, int tokens, cudaStream_t s) {
  return p.a.heads <= 16 ? launch_latent<NS, VS, 1>(tc, p, tokens, s) : launch_latent<NS, VS, 2>(tc, p, tokens, s);
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

extern "C" long long nkb_latent_scratch_floats(const NkbLatentArgs* a, int tokens, int num_splits) {
  int vs = 0;
  if (num_splits <= 1 || !latent_shape(*a, &vs)) return 0;
  const int rows = a->heads <= 16 ? 16 : 32;
  return kLatCounters + (long long)tokens * ((a->heads + rows - 1) / rows) * num_splits * (rows * vs * 64 + 2 * rows);
}

// Attention of new tokens, already in the cache, over the visible cached rows; queries and results as latents, bf16.  q_lens null:
// token t belongs to sequence t.  Returns -5 for sizes it does not take.
extern "C" int nkb_latent_attn(const NkbLatentArgs* a, const void* q, const void* cache, const int* block_table,
                               const int* q_start, const int* q_lens, const int* context_lens, void* out, float* scratch,
                               int batch, int tokens, int block_size, int num_blocks, int max_blocks_per_seq, int num_splits,
                               void* stream) {
  if (batch <= 0 || tokens <= 0) return 0;
  int vs = 0;
  const int ns = latent_shape(*a, &vs);
  if (!ns || a->row != ns * 64) return -5;
  if (!latent_ok(*a) || block_size != kLatPage || tokens > 65535 || (!q_lens && tokens != batch)) return -2;
  if ((reinterpret_cast<uintptr_t>(q) & 3) || ((a->q_token | a->q_head) & 1) || (reinterpret_cast<uintptr_t>(out) & 3)) return -2;
  if (!status_word() && nkb_init() != 0) return -1;
  LatentMmaParams p{};
  p.a = *a;
  const int rows = a->heads <= 16 ? 16 : 32;
  if (num_splits < 1) num_splits = 1;
  if (num_splits > 1 && (!scratch || (long long)tokens * ((a->heads + rows - 1) / rows) > kLatCounters)) return -2;
  p.q = reinterpret_cast<const __nv_bfloat16*>(q);
  p.block_table = block_table; p.q_start = q_start; p.q_lens = q_lens; p.context_lens = context_lens;
  p.out = reinterpret_cast<__nv_bfloat16*>(out);
  p.scratch = num_splits > 1 ? scratch + kLatCounters : scratch;
  p.counters = reinterpret_cast<unsigned int*>(scratch);
  p.status = status_word();
  p.batch = batch; p.max_blocks = max_blocks_per_seq; p.num_splits = num_splits;
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
