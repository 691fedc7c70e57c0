// Blockwise prefill attention with two score maps over shared values (differential attention, attn_maps.h) on
// tcgen05 for sm_100a, over the paged cache.
//
// One CTA per (128 query rows, query head, sequence).  The structure is that of attn_prefill.cu with the two maps of
// the head in the place of its two query tiles: each map has its own scores S_t = Q_t K_t^T and probabilities and its
// own accumulator O_t += P_t V in tensor memory, both maps read the same V tile, and the epilogue combines O_0 and
// O_1 (o = a_0 - lambda a_1, root-mean-square norm over the head) without either leaving the chip.
//   warp 0     TMA producer: the Q tile once, then a ring of 128-token K and V tiles.  A key row holds both
//              maps' keys side by side, so one K tile serves both; map t's contraction steps are the t-th half of it.
//   warps 1, 2 MMA issuers, one per map
//   warps 4-7  softmax of map 0, warps 8-11 of map 1, one thread per query row, exponentials in turns
//
// The score cap softcap * tanh(s / softcap) is evaluated in fp32: on rows whose scores all stay below 0.6 softcap
// as an odd polynomial on the FMA pipe (least-squares fit at Chebyshev nodes, relative error 3e-9), otherwise as
// 1 - 2 / (exp(2 y) + 1).  The special-function unit is the bottleneck of this kernel, and the second form needs it
// three times per score instead of once.
#include "common.cuh"
#include "attn_maps.h"
#include "api.h"
#include <math.h>

namespace nkb {

constexpr int kMpTile = 128;
constexpr int kMpPage = 32;
constexpr int kMpThreads = 384;
constexpr float kMpRescaleStep = 8.f;
constexpr float kMpPolyLimit = 0.6f;

struct MapsPrefillParams {
  NkbMapsArgs a;
  const int* block_table;
  const int* q_start;
  const int* q_lens;
  const int* context_lens;
  __nv_bfloat16* out;
  int* status;
  int max_blocks;
};

template <int STAGES>
struct MapsPrefillCtrl {
  uint64_t q_full;
  uint64_t kv_full[STAGES], kv_empty[STAGES];
  uint64_t s_full[2], s_empty[2];
  uint64_t p_full[2], o_full[2];
  uint64_t turn[2][4];
  float l1[kMpTile];
  uint32_t tmem_base;
  int abort;
};

__device__ __noinline__ bool mp_wait_slow(uint64_t* bar, uint32_t parity, volatile int* abort_flag, int* status, int code) {
  return mbar_wait(bar, parity, abort_flag, status, code);
}
__device__ __forceinline__ bool mp_wait(uint64_t* bar, uint32_t parity, volatile int* abort_flag, int* status, int code) {
  if (mbar_try_wait(bar, parity)) return true;
  return mp_wait_slow(bar, parity, abort_flag, status, code);
}

__device__ __forceinline__ float2 dup2(float x) { return make_float2(x, x); }

// DP: padded size of one map's query / key (32 or 64), VD: padded value size (64 or 128)
template <int DP, int VD>
__global__ void __launch_bounds__(kMpThreads, 1)
maps_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                    const __grid_constant__ CUtensorMap tmV, const __grid_constant__ MapsPrefillParams p) {
  constexpr int NK = 2 * DP / 64, NV = VD / 64;
  constexpr int kHalf = 128 * 128;                       // [128 rows][64 bf16] swizzled slab
  constexpr int kStageBytes = (NK > NV ? NK : NV) * kHalf;
  constexpr int kPBytes = 2 * kHalf;
  constexpr int kStages = 4;
  constexpr int kSteps = DP / 16;                        // contraction steps of one map
  constexpr uint32_t kTmemCols = 512, kSCol = 0, kOCol = 256;
  using Ctrl = MapsPrefillCtrl<kStages>;

  const int qt = gridDim.x - 1 - blockIdx.x, head = blockIdx.y, b = blockIdx.z;
  griddep_wait();
  griddep_launch();
  const int q_len = p.q_lens[b];
  if (qt * kMpTile >= q_len) return;
  const int ctx = p.context_lens[b];
  if (ctx < q_len) return;                               // inactive row
  const int q_row0 = p.q_start[b] + qt * kMpTile;
  const int kvh = head / (p.a.heads / p.a.kv_heads);
  const int rows = min(kMpTile, q_len - qt * kMpTile);
  const int pos0 = ctx - q_len + qt * kMpTile;
  const int n_tiles = (pos0 + rows - 1) / kMpTile + 1;   // tiles up to the diagonal; at least one

  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* q_s = smem;
  uint8_t* kv_s = q_s + NK * kHalf;
  uint8_t* p_s = kv_s + kStages * kStageBytes;
  Ctrl* ctrl = reinterpret_cast<Ctrl*>(p_s + 2 * kPBytes);
  const int warp = warp_idx_uniform(), lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
    mbar_init(&ctrl->q_full, 1);
    for (int i = 0; i < kStages; ++i) {
      mbar_init(&ctrl->kv_full[i], 1);
      mbar_init(&ctrl->kv_empty[i], 2);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&ctrl->s_full[i], 1);
      mbar_init(&ctrl->s_empty[i], 4);
      mbar_init(&ctrl->p_full[i], 4);
      mbar_init(&ctrl->o_full[i], 1);
      for (int q = 0; q < 4; ++q) mbar_init(&ctrl->turn[i][q], 1);
    }
    ctrl->abort = 0;
    mbar_fence_init();
    fence_proxy_async();
  }
  if (warp == 1) {
    tmem_alloc(&ctrl->tmem_base, kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = __shfl_sync(0xffffffffu, ctrl->tmem_base, 0);
  volatile int* abort_flag = &ctrl->abort;

  if (warp == 0) {
    // ---------------------------------------------------------------- TMA producer
    if (lane == 0) {
      mbar_expect_tx(&ctrl->q_full, NK * kHalf);
#pragma unroll
      for (int h = 0; h < NK; ++h) tma_load_3d(q_s + h * kHalf, &tmQ, &ctrl->q_full, h * 64, head, q_row0);
    }
    __syncwarp();
    const int* table = p.block_table + (long long)b * p.max_blocks;
    const int last_page = max((ctx + kMpPage - 1) / kMpPage - 1, 0);
    int seq = 0;
    bool live = true;
    // ring order: K(0), then per tile u: K(u + 1), V(u)
    auto load = [&](bool is_v, int j) {
      if (!live) return;
      const int st = seq % kStages;
      const uint32_t ph = uint32_t(seq / kStages) & 1u;
      ++seq;
      bool ok = mp_wait(&ctrl->kv_empty[st], ph ^ 1u, abort_flag, p.status, ERR_WAIT_SMEM_EMPTY);
      if (!__all_sync(0xffffffffu, ok)) { live = false; return; }
      int blk[4];
#pragma unroll
      for (int pi = 0; pi < 4; ++pi) blk[pi] = table[min(j * 4 + pi, last_page)];
      if (lane == 0) {
        uint8_t* dst = kv_s + st * kStageBytes;
        const int slabs = is_v ? NV : NK;
        mbar_expect_tx(&ctrl->kv_full[st], slabs * kHalf);
        for (int pi = 0; pi < 4; ++pi)
          for (int h = 0; h < slabs; ++h)
            tma_load_4d(dst + h * kHalf + pi * (kMpPage * 128), is_v ? &tmV : &tmK, &ctrl->kv_full[st], h * 64, 0, kvh,
                        blk[pi]);
      }
      __syncwarp();
    };
    load(false, 0);
#pragma unroll 1
    for (int u = 0; u < n_tiles && live; ++u) {
      if (u + 1 < n_tiles) load(false, u + 1);
      load(true, u);
    }
  } else if (warp == 1 || warp == 2) {
    // ---------------------------------------------------------------- MMA issuers, one per map
    constexpr uint32_t idesc_qk = make_idesc_bf16(128, kMpTile, 0, 0);
    constexpr uint32_t idesc_pv = make_idesc_bf16(128, VD, 0, 1);
    const int t = warp - 1;
    const uint32_t q_lo = uint32_t(make_smem_desc_sw128(smem_u32(q_s), 0, 1024));
    const uint32_t kv_lo = uint32_t(make_smem_desc_sw128(smem_u32(kv_s), 0, 1024));
    const uint32_t p_lo = uint32_t(make_smem_desc_sw128(smem_u32(p_s + t * kPBytes), 0, 1024));
    const uint64_t hk = uint64_t(uint32_t(make_smem_desc_sw128(0, 0, 1024) >> 32)) << 32;
    const uint32_t lbo_v = (uint32_t(kHalf) >> 4) << 16;
    const uint32_t s_tmem = tmem_base + kSCol + t * 128, o_tmem = tmem_base + kOCol + t * 128;
    if (elect_one()) {
      bool ok = mp_wait(&ctrl->q_full, 0, abort_flag, p.status, ERR_WAIT_SMEM_FULL);
      int seq = 0;
      auto do_k = [&](int x) {
        if (x >= n_tiles || !ok) return;
        const int item = seq++, st = item % kStages;
        ok = mp_wait(&ctrl->kv_full[st], uint32_t(item / kStages) & 1u, abort_flag, p.status, ERR_WAIT_SMEM_FULL);
        if (!ok) return;
        ok = mp_wait(&ctrl->s_empty[t], (uint32_t(x) & 1u) ^ 1u, abort_flag, p.status, ERR_WAIT_TMEM_EMPTY);
        if (!ok) return;
        tc_fence_after();
        const uint32_t kvd = kv_lo + uint32_t(st * kStageBytes >> 4);
        uint64_t da[kSteps], db[kSteps];
#pragma unroll
        for (int s = 0; s < kSteps; ++s) {
          const int gk = t * kSteps + s;                 // 16-wide step of the whole key row
          const uint32_t off = uint32_t((gk >> 2) * (kHalf >> 4) + (gk & 3) * 2);
          da[s] = hk | (q_lo + off);
          db[s] = hk | (kvd + off);
        }
#pragma unroll
        for (int s = 0; s < kSteps; ++s) umma_f16(s_tmem, da[s], db[s], idesc_qk, s > 0 ? 1u : 0u);
        umma_commit(&ctrl->s_full[t]);
        umma_commit(&ctrl->kv_empty[st]);
      };
      auto do_v = [&](int x) {
        if (!ok) return;
        const int item = seq++, st = item % kStages;
        ok = mp_wait(&ctrl->kv_full[st], uint32_t(item / kStages) & 1u, abort_flag, p.status, ERR_WAIT_SMEM_FULL);
        if (!ok) return;
        ok = mp_wait(&ctrl->p_full[t], uint32_t(x) & 1u, abort_flag, p.status, ERR_WAIT_SOFTMAX);
        if (!ok) return;
        tc_fence_after();
        const uint32_t kvd = kv_lo + uint32_t(st * kStageBytes >> 4);
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          uint64_t da[4], db[4];
#pragma unroll
          for (int k4 = 0; k4 < 4; ++k4) {
            db[k4] = hk | ((kvd + uint32_t((h * 4 + k4) * 128)) | lbo_v);
            da[k4] = hk | (p_lo + uint32_t(h * (kHalf >> 4) + k4 * 2));
          }
#pragma unroll
          for (int k4 = 0; k4 < 4; ++k4) umma_f16(o_tmem, da[k4], db[k4], idesc_pv, (x > 0 || h > 0 || k4 > 0) ? 1u : 0u);
        }
        umma_commit(&ctrl->o_full[t]);
        umma_commit(&ctrl->kv_empty[st]);
      };
      do_k(0);
#pragma unroll 1
      for (int u = 0; u < n_tiles && ok; ++u) {
        do_k(u + 1);
        do_v(u);
      }
    }
    __syncwarp();
  } else if (warp >= 4) {
    // ---------------------------------------------------------------- softmax
    const int t = (warp - 4) >> 2;
    const int quad = warp & 3;
    const int r = quad * 32 + lane;
    const int q_pos = pos0 + r;
    const uint32_t lane_off = uint32_t(quad * 32) << 16;
    const uint32_t s_addr = tmem_base + lane_off + kSCol + t * 128;
    const uint32_t o_addr = tmem_base + lane_off + kOCol + t * 128;
    uint8_t* my_p = p_s + t * kPBytes + r * 128;
    const bool capped = p.a.softcap > 0.f;
    constexpr float kLog2e = 1.4426950408889634f;
    // uncapped: scores are scaled to the log2 domain in the exponential's multiply-add; capped: already there
    const float sc = capped ? 1.f : p.a.scale * kLog2e;
    const float inv_cap = capped ? 1.f / p.a.softcap : 0.f;
    const float k_y = p.a.scale * inv_cap;               // raw score -> argument of tanh
    const float cap2 = p.a.softcap * kLog2e;
    const float poly_raw = capped ? kMpPolyLimit / fmaxf(fabsf(k_y), 1e-30f) : 0.f;
    float m = -INFINITY, l = 0.f;
    const int hi_pos = min(ctx - 1, q_pos);
    bool alive = true;

    for (int it = 0; it < n_tiles; ++it) {
      const int kv0 = it * kMpTile;
      bool ok = mp_wait(&ctrl->s_full[t], uint32_t(it) & 1u, abort_flag, p.status, ERR_WAIT_TMEM_FULL);
      if (!__all_sync(0xffffffffu, ok)) { alive = false; break; }
      tc_fence_after();
      uint32_t v[kMpTile];
#pragma unroll
      for (int c = 0; c < kMpTile / 32; ++c) tmem_ld_32x32(s_addr + c * 32, reinterpret_cast<uint32_t(&)[32]>(v[c * 32]));
      tmem_ld_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&ctrl->s_empty[t]);

      if (capped) {
        float mx4[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) mx4[i] = fmaxf(fabsf(__uint_as_float(v[2 * i])), fabsf(__uint_as_float(v[2 * i + 1])));
#pragma unroll
        for (int i = 8; i < kMpTile; i += 2)
          mx4[(i >> 1) & 3] = fmax3(mx4[(i >> 1) & 3], fabsf(__uint_as_float(v[i])), fabsf(__uint_as_float(v[i + 1])));
        const float am = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
        if (__all_sync(0xffffffffu, am <= poly_raw)) {
          // y * P(y^2), P(u) ~ tanh(sqrt(u)) / sqrt(u) on [0, 0.36]
          const float2 ky2 = dup2(k_y), c2 = dup2(cap2);
#pragma unroll
          for (int i = 0; i < kMpTile; i += 2) {
            const float2 y = fmul2(make_float2(__uint_as_float(v[i]), __uint_as_float(v[i + 1])), ky2);
            const float2 u = fmul2(y, y);
            float2 q = ffma2(u, dup2(-0.005856427870f), dup2(0.020757475450f));
            q = ffma2(q, u, dup2(-0.053769921786f));
            q = ffma2(q, u, dup2(0.133317047022f));
            q = ffma2(q, u, dup2(-0.333332839718f));
            q = ffma2(q, u, dup2(0.999999997563f));
            const float2 w = fmul2(fmul2(y, c2), q);
            v[i] = __float_as_uint(w.x);
            v[i + 1] = __float_as_uint(w.y);
          }
        } else {
          const float k_e = 2.f * kLog2e * k_y;
#pragma unroll
          for (int i = 0; i < kMpTile; ++i) {
            const float e = exp2f(__uint_as_float(v[i]) * k_e);
            v[i] = __float_as_uint(fmaf(-2.f * cap2, __fdividef(1.f, e + 1.f), cap2));
          }
        }
      }
      if (__any_sync(0xffffffffu, kv0 + kMpTile - 1 > hi_pos)) {
        const int hi_rel = hi_pos - kv0;
#pragma unroll
        for (int i = 0; i < kMpTile; ++i)
          if (i > hi_rel) v[i] = 0xff800000u;
      }
      float mx4[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) mx4[i] = fmaxf(__uint_as_float(v[2 * i]), __uint_as_float(v[2 * i + 1]));
#pragma unroll
      for (int i = 8; i < kMpTile; i += 2)
        mx4[(i >> 1) & 3] = fmax3(mx4[(i >> 1) & 3], __uint_as_float(v[i]), __uint_as_float(v[i + 1]));
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * sc;

      bool p_free = it == 0;
      if (it == 0) {
        m = mx;
      } else {
        const bool grow = mx > m + kMpRescaleStep || (m == -INFINITY && mx > -INFINITY);
        if (__any_sync(0xffffffffu, grow)) {
          ok = mp_wait(&ctrl->o_full[t], uint32_t(it - 1) & 1u, abort_flag, p.status, ERR_WAIT_TMEM_FULL);
          if (!__all_sync(0xffffffffu, ok)) { alive = false; break; }
          p_free = true;
          tc_fence_after();
          const float alpha = grow ? exp2f(m - mx) : 1.f;
#pragma unroll 1
          for (int c = 0; c < VD / 32; ++c) {
            uint32_t o[32];
            tmem_ld_32x32(o_addr + c * 32, o);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
            tmem_st_32x32(o_addr + c * 32, o);
          }
          tmem_st_wait();
          l *= alpha;
          if (grow) m = mx;
        }
      }
      const float base = (m == -INFINITY) ? 0.f : m;
      const float2 sc2 = dup2(sc), nb2 = dup2(-base);
      float2 sum2[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) sum2[i] = dup2(0.f);
      if (!p_free) {
        ok = mp_wait(&ctrl->o_full[t], uint32_t(it - 1) & 1u, abort_flag, p.status, ERR_WAIT_TMEM_FULL);
        if (!__all_sync(0xffffffffu, ok)) { alive = false; break; }
      }
      // the maps' exponentials take turns on the special-function unit (see attn_prefill.cu)
      if (t == 1 || it >= 1) {
        ok = mp_wait(&ctrl->turn[t][quad], uint32_t(t == 0 ? it - 1 : it) & 1u, abort_flag, p.status, ERR_WAIT_SOFTMAX);
        if (!__all_sync(0xffffffffu, ok)) { alive = false; break; }
      }
#pragma unroll
      for (int c = 0; c < kMpTile / 32; ++c) {
        uint32_t pk[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const int k = c * 32 + 2 * i;
          const float2 x = ffma2(make_float2(__uint_as_float(v[k]), __uint_as_float(v[k + 1])), sc2, nb2);
          const float2 e = make_float2(exp2f(x.x), exp2f(x.y));
          sum2[i & 3] = fadd2(sum2[i & 3], e);
          pk[i] = pack_bf16x2(e.x, e.y);
        }
#pragma unroll
        for (int q = 0; q < 4; ++q)
          *reinterpret_cast<uint4*>(my_p + (c >> 1) * kHalf + ((((c & 1) * 4 + q) ^ (r & 7)) << 4)) =
              make_uint4(pk[4 * q], pk[4 * q + 1], pk[4 * q + 2], pk[4 * q + 3]);
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&ctrl->turn[1 - t][quad]);
      fence_proxy_async();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&ctrl->p_full[t]);
      {
        const float2 s01 = fadd2(sum2[0], sum2[1]), s23 = fadd2(sum2[2], sum2[3]);
        const float2 s4 = fadd2(s01, s23);
        l += s4.x + s4.y;
      }
    }
    // ---- epilogue: map 0's warps combine both accumulators.  The barrier comes first: past it map 1's warps have
    // seen all but the last phase of their o_full, so waiting for that phase's parity cannot match an older one.
    if (t == 1) ctrl->l1[r] = l;
    asm volatile("bar.sync 1, 256;" ::: "memory");
    if (t == 0) {
      bool ok = alive && mp_wait(&ctrl->o_full[0], uint32_t(n_tiles - 1) & 1u, abort_flag, p.status, ERR_WAIT_TMEM_FULL) &&
                mp_wait(&ctrl->o_full[1], uint32_t(n_tiles - 1) & 1u, abort_flag, p.status, ERR_WAIT_TMEM_FULL);
      if (__all_sync(0xffffffffu, ok) && !*abort_flag) {
        tc_fence_after();
        const float i0 = 1.f / l, i1 = p.a.lambda / ctrl->l1[r];
        float x[VD];
        float ss = 0.f;
#pragma unroll
        for (int c = 0; c < VD / 32; ++c) {
          uint32_t a[32], d[32];
          tmem_ld_32x32(o_addr + c * 32, a);
          tmem_ld_32x32(o_addr + 128 + c * 32, d);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            x[c * 32 + i] = __uint_as_float(a[i]) * i0 - __uint_as_float(d[i]) * i1;
            ss += x[c * 32 + i] * x[c * 32 + i];
          }
        }
        if (r < rows) {
          const float inv = p.a.out_scale / sqrtf(ss / float(p.a.vdim) + p.a.eps);
          __nv_bfloat16* dst = p.out + ((long long)(q_row0 + r) * p.a.heads + head) * p.a.vdim;
          if ((p.a.vdim & 7) == 0) {
#pragma unroll
            for (int i = 0; i < VD; i += 8) {
              if (i < p.a.vdim)
                *reinterpret_cast<uint4*>(dst + i) =
                    make_uint4(pack_bf16x2(x[i] * inv, x[i + 1] * inv), pack_bf16x2(x[i + 2] * inv, x[i + 3] * inv),
                               pack_bf16x2(x[i + 4] * inv, x[i + 5] * inv), pack_bf16x2(x[i + 6] * inv, x[i + 7] * inv));
            }
          } else {
#pragma unroll
            for (int i = 0; i < VD; ++i)
              if (i < p.a.vdim) dst[i] = __float2bfloat16(x[i] * inv);
          }
        }
      }
    }
  }

  if (*abort_flag) {
    for (int i = 0; i < 200; ++i) __nanosleep(1000);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, kTmemCols);
  }
}

template <int DP, int VD>
static int launch_maps_prefill(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv,
                               const MapsPrefillParams& p, int batch, int max_q_len, cudaStream_t s) {
  constexpr int NK = 2 * DP / 64, NV = VD / 64, kStageSlabs = NK > NV ? NK : NV;
  constexpr int smem = 16384 * (NK + 4 * kStageSlabs + 4) + int(sizeof(MapsPrefillCtrl<4>)) + 1024;
  static_assert(smem <= 232448, "shared memory of one CTA");
  static bool attr_set[64] = {false};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -1;
  if (!attr_set[dev]) {
    cudaError_t e = cudaFuncSetAttribute(maps_prefill_kernel<DP, VD>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return int(e);
    attr_set[dev] = true;
  }
  const dim3 grid((max_q_len + kMpTile - 1) / kMpTile, p.a.heads, batch);
  return launch_pdl(maps_prefill_kernel<DP, VD>, grid, dim3(kMpThreads), size_t(smem), s, tq, tk, tv, p);
}

}  // namespace nkb

using namespace nkb;

// q [total_q, heads, 2 * dim_p] packs the new tokens of all sequences (rotated, already appended to the cache); out
// [total_q, heads * vdim].  Two maps, dim_p 32 or 64, vdim_p 64 or 128; -5 for sizes it does not take.
extern "C" int nkb_maps_attn_prefill(const NkbMapsArgs* a, const void* q, const void* k_cache, const void* v_cache,
                                     const int* block_table, const int* q_start, const int* q_lens,
                                     const int* context_lens, void* out, int batch, int total_q, int max_q_len,
                                     int block_size, int num_blocks, int max_blocks_per_seq, void* stream) {
  if (batch <= 0 || total_q <= 0) return 0;
  if (a->maps != 2 || a->window > 0 || (a->dim_p != 32 && a->dim_p != 64) || (a->vdim_p != 64 && a->vdim_p != 128)) return -5;
  if (block_size != kMpPage || a->kv_heads < 1 || a->heads % a->kv_heads || batch > 65535 || a->heads > 65535) return -2;
  if (!status_word() && nkb_init() != 0) return -1;
  MapsPrefillParams p{};
  p.a = *a;
  p.block_table = block_table; p.q_start = q_start; p.q_lens = q_lens; p.context_lens = context_lens;
  p.out = reinterpret_cast<__nv_bfloat16*>(out);
  p.status = status_word();
  p.max_blocks = max_blocks_per_seq;
  const int kw = 2 * a->dim_p;
  CUtensorMap tq, tk, tv;
  {
    const uint64_t dims[3] = {uint64_t(kw), uint64_t(a->heads), uint64_t(total_q)};
    const uint64_t strides[2] = {uint64_t(kw) * 2, uint64_t(kw) * a->heads * 2};
    const uint32_t box[3] = {64, 1, uint32_t(kMpTile)};
    if (encode_tmap_bf16(&tq, q, 3, dims, strides, box)) return -4;
  }
  auto encode = [&](CUtensorMap* m, const void* ptr, int width) {
    const uint64_t dims[4] = {uint64_t(width), uint64_t(kMpPage), uint64_t(a->kv_heads), uint64_t(num_blocks)};
    const uint64_t strides[3] = {uint64_t(width) * 2, uint64_t(width) * kMpPage * 2,
                                 uint64_t(width) * kMpPage * a->kv_heads * 2};
    const uint32_t box[4] = {64, uint32_t(kMpPage), 1, 1};
    return encode_tmap_bf16(m, ptr, 4, dims, strides, box);
  };
  if (encode(&tk, k_cache, kw) || encode(&tv, v_cache, a->vdim_p)) return -4;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dim_p == 32 && a->vdim_p == 64) return launch_maps_prefill<32, 64>(tq, tk, tv, p, batch, max_q_len, s);
  if (a->dim_p == 32) return launch_maps_prefill<32, 128>(tq, tk, tv, p, batch, max_q_len, s);
  if (a->vdim_p == 64) return launch_maps_prefill<64, 64>(tq, tk, tv, p, batch, max_q_len, s);
  return launch_maps_prefill<64, 128>(tq, tk, tv, p, batch, max_q_len, s);
}
