// Blockwise (flash) prefill attention on tcgen05 for sm_100a, reading K/V from
// the paged cache through the per-sequence block table.
//
// One CTA per (256 query rows, query head, sequence), as two 128-row query tiles in ping-pong:
//   warp 0     TMA producer: both Q tiles once, then a 3-stage ring of 128-token K and V tiles (four
//              32-token pages each, 128-byte swizzle, non-multicast)
//   warps 1, 2 issue tcgen05.mma, one warp per query tile t, per KV tile j in the order
//              S_t(j+1) = Q_t K(j+1)^T, then O_t += P_t(j) V(j) (V is an MN-major B operand).  S_t is free
//              as soon as the softmax holds it in registers, so the next scores are ready when the
//              softmax of tile j ends and the softmax warps do not wait for the tensor pipe.
//   warps 4-7  softmax of tile 0, warps 8-11 softmax of tile 1: one thread per query row reads its
//              128 scores from TMEM once, keeps them in registers, and writes P as bf16 to shared memory
//              in the swizzled K-major layout the MMA reads.  The two tiles take turns with their
//              exponentials (see the loop), so that one tile's MMAs, score loads and row maxima run
//              while the other tile has the special-function unit.
// O_0 and O_1 stay in TMEM for the whole KV loop (S_0, S_1, O_0, O_1 = 4 x 128 columns).  The row maximum
// that scales the exponentials is only raised when the true maximum has grown by more than 2^8 since it
// was last set; then the row's O is rescaled in TMEM (load, multiply, store).  With a stale maximum the
// probabilities are at most 2^8 too large, which fp32 sums and bf16 P hold without loss, and O / l is
// unchanged because both carry the same factor.  KV tiles past a query tile's causal diagonal or before
// its window are skipped for that tile; the mask is only evaluated on tiles that cross either edge.
// GQA needs no repeat of K/V: the query head picks its kv head.  Supports causal
// masking with a cached prefix (q_len <= context_len), sliding windows, chunks and
// attention-sink logits.
//
// Keys wider than values (latent attention): the sizes are counted in slabs of 64 columns, NK of queries and keys and NV of
// values, KT tokens per KV tile (64 with three slabs, to fit shared memory).  In the ROWS form K and V are not paged: token j of
// sequence b is row kv_base[b] + j of matrices with one column block per head, and the last slab of every head's keys
// comes from a matrix that all heads share (the rotated key part).
//
// What the structure answers to (measured on B200 with a cycle trace of one CTA and an issue-rate probe):
// * The tensor pipe runs a 128 x 128 x 16 MMA in 64 cycles from any operand source, but queues only a few of
//   them: whatever the issuing thread does between two groups of MMAs is time in which the pipe drains.  A single
//   thread runs one dependent instruction every few cycles, and a blocking wait for one query tile kept the
//   other tile's ready group from being issued.  Hence one issuer per query tile, issue by a single elected
//   thread without warp votes, descriptors prepared before four MMAs go out as one instruction sequence, and
//   warp roles the compiler can prove uniform.
// * 128 exponentials per row keep the special-function unit of a scheduler busy for about as long as the rest
//   of an iteration takes.  Left alone, the two query tiles fall into step (they share the K/V ring), compute
//   their exponentials at half speed at the same time and then wait at the same time.
// * Computing part of the exponentials with a polynomial on the FMA pipe, a branch per 32 scores in the
//   exponential loop (to skip fully masked groups) and probabilities in tensor memory (which ties Q K^T of
//   the next tile to P V of this one) were all measured slower than what is here.
//
// Reference parity: prefill branch of attention_kernel in
// examples/models/qwen3/kernels/attention.py:108-137 (materialised scores +
// additive -1e5 mask + softmax + P.V), window / sinks from
// examples/models/gpt_oss/kernels/attention.py:116-148, non-causal-free prefill
// of examples/models/qwen3_embedding/kernels/attention.py.
#include "common.cuh"
#include "attn_maps.h"
#include "api.h"
#include <math.h>

namespace nkb {

constexpr int kQTile = 128;          // rows of one MMA tile
constexpr int kQPair = 2 * kQTile;   // query rows per CTA
constexpr int kPfPage = 32;
constexpr int kPfThreads = 384;      // warpgroup 0: TMA warp, two MMA warps, one idle; warpgroups 1, 2: softmax
constexpr int kMaxKVStages = 4;
constexpr float kRescaleStep = 8.f;  // log2 of the growth of the row maximum that triggers a rescale of O

struct PrefillParams {
  const int* block_table;
  const int* q_start;
  const int* q_lens;
  const int* context_lens;
  __nv_bfloat16* out;
  const float* sinks;
  const int* kv_base;                  // ROWS: row of position 0 of every sequence (may be negative)
  int* status;
  int nq, nkv, max_blocks, causal, window, chunk;
  float scale_log2;
  NkbScoreMods mods;                   // MODS only
  int dist_far;                        // > 0: the terms up to this distance are a table in shared memory
};

struct PrefillCtrl {
  uint64_t q_full;
  uint64_t kv_full[kMaxKVStages], kv_empty[kMaxKVStages];
  uint64_t s_full[2], s_empty[2];
  uint64_t p_full[2], o_full[2];
  uint64_t turn[2][4];
  uint32_t tmem_base;
  int abort;
};

// Bounded barrier wait whose slow path (timer, abort flag) is one shared out-of-line function: the kernel has two
// dozen waits and their inlined loops would push the hot code out of the instruction cache.
__device__ __noinline__ bool pf_wait_slow(uint64_t* bar, uint32_t parity, volatile int* abort_flag, int* status,
                                          int code) {
  return mbar_wait(bar, parity, abort_flag, status, code);
}
__device__ __forceinline__ bool pf_wait(uint64_t* bar, uint32_t parity, volatile int* abort_flag, int* status,
                                        int code) {
  if (mbar_try_wait(bar, parity)) return true;
  return pf_wait_slow(bar, parity, abort_flag, status, code);
}

// KV tile range [lo, hi) that query tile `t` of the CTA attends to (empty when the tile has no rows).
struct TileRange {
  int lo, hi, pos0, rows;
};
template <int kKVTile>
__device__ __forceinline__ TileRange tile_range(const PrefillParams& p, int row0, int q_len, int ctx) {
  TileRange r{0, 0, 0, 0};
  if (row0 >= q_len) return r;
  r.rows = min(kQTile, q_len - row0);
  r.pos0 = ctx - q_len + row0;                       // kv position of the tile's first query
  r.hi = (ctx + kKVTile - 1) / kKVTile;
  if (p.causal) r.hi = min(r.hi, (r.pos0 + r.rows - 1) / kKVTile + 1);
  r.lo = nkb_first_visible(r.pos0, p.window, p.chunk) / kKVTile;
  if (r.hi < r.lo) r.hi = r.lo;
  return r;
}

template <int NK, int NV, int KT>
struct PrefillSmem {
  static constexpr int kHalf = kQTile * 128;          // [128 rows][64 bf16] swizzled slab = 16 KB
  static constexpr int kKVHalf = KT * 128;            // slab of a K or V tile
  static constexpr int kQBytes = NK * kHalf;          // one query tile
  static constexpr int kStageBytes = (NK > NV ? NK : NV) * kKVHalf;
  static constexpr int kPBytes = KT / 64 * kHalf;     // [128 rows][KT tokens]
  static constexpr int kStages = NK == 3 || KT == 64 ? 4 : 3;
  static constexpr int kBytes = 2 * kQBytes + kStages * kStageBytes + 2 * kPBytes + int(sizeof(PrefillCtrl)) + 1024 + 64;
  // Table of the distance term: element j of a copy belongs to distance far - j.  Tiles that a query tile walks hold distances from
  // -(126 + KT) to window + KT + 253.  Copy c starts c elements later, so that four scores of any row are one aligned access;
  // its pitch spreads the copies over the banks.
  static __host__ __device__ constexpr int far_of(int window) { return window + KT + 256; }
  static __host__ __device__ constexpr int pitch_of(int far) { return (far + KT + 128 + 4 + 31) / 32 * 32 + 8; }
};

// MODS: scores are capped, lose a term that grows with the distance, or the first tokens stay visible outside the window.
// The special-function unit is the bottleneck of the softmax, so that it should see no more than one operation per score: the cap is
// an odd polynomial where all scores of a row stay below 0.35 or 1.1 of it (fits at Chebyshev nodes, relative errors 4e-8 and 2e-8;
// beyond, the exponential form), and the distance term is read from a table wherever a window bounds the distances.
template <int NK, int NV, int KT, bool ROWS, bool MODS>
__global__ void __launch_bounds__(kPfThreads, 1)
flash_attn_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                          const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmR,
                          const PrefillParams p) {
  using L = PrefillSmem<NK, NV, KT>;
  constexpr int D = NV * 64, kKVTile = KT, kHalf = L::kHalf, kKVHalf = L::kKVHalf, kQBytes = L::kQBytes;
  constexpr int kKVBytes = L::kStageBytes, kPBytes = L::kPBytes, kKVStages = L::kStages;
  constexpr uint32_t kTmemCols = 512;
  constexpr uint32_t kSCol = 0, kOCol = 256;   // S_t at kSCol + 128 t, O_t at kOCol + 128 t

  // the heaviest CTAs (last query rows of a causal sequence) start first
  const int qt = gridDim.x - 1 - blockIdx.x, head = blockIdx.y, b = blockIdx.z;
  griddep_wait();
  griddep_launch();
  const int q_len = p.q_lens[b];
  if (qt * kQPair >= q_len) return;
  const int ctx = p.context_lens[b];
  const int q_row0 = p.q_start[b] + qt * kQPair;        // row in the packed q / out arrays
  const int kvh = head / (p.nq / p.nkv);
  const TileRange tr0 = tile_range<KT>(p, qt * kQPair, q_len, ctx);
  TileRange tr1 = tile_range<KT>(p, qt * kQPair + kQTile, q_len, ctx);
  const bool two = tr1.rows > 0;
  // union of the two ranges; every tile of it is attended to by at least one query tile
  const int u_lo = tr0.lo, u_hi = two ? max(tr0.hi, tr1.hi) : tr0.hi;
  // KV tiles of kept first tokens come ahead of the union (those that are not in it).  Where they reach into it, the second query
  // tile walks all of the union: a tile it sees nothing of is masked.
  int kept = 0;
  if constexpr (MODS) {
    kept = (p.mods.keep_first + KT - 1) / KT;
    if (kept > u_lo) {
      kept = u_lo;
      if (two) tr1.lo = u_lo;
    }
  }
  const int n_union = kept + u_hi - u_lo;
  const auto tile_at = [&](int x) { return MODS && x < kept ? x : x - kept + u_lo; };     // KV tile of walk position x

  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* q_s = smem;                              // 2 query tiles
  uint8_t* kv_s = q_s + 2 * kQBytes;                // ring of K and V tiles
  uint8_t* p_s = kv_s + kKVStages * kKVBytes;       // 2 probability tiles
  PrefillCtrl* ctrl = reinterpret_cast<PrefillCtrl*>(p_s + 2 * kPBytes);

  const int warp = warp_idx_uniform(), lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
    if constexpr (ROWS) tma_prefetch_desc(&tmR);
    mbar_init(&ctrl->q_full, 1);
    for (int i = 0; i < kKVStages; ++i) {
      mbar_init(&ctrl->kv_full[i], 1);
      mbar_init(&ctrl->kv_empty[i], two ? 2 : 1);   // one release from each query tile's issuer
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
  if constexpr (MODS) {
    if (p.dist_far > 0) {
      const float da = p.mods.dist_a[head], db = p.mods.dist_b[head];
      float* tab = reinterpret_cast<float*>(ctrl + 1);
      const int pitch = L::pitch_of(p.dist_far);
      for (int j = threadIdx.x; j < pitch + 3; j += kPfThreads) {
        const float x = -da * __log2f(fmaf(db, float(max(p.dist_far - j, 0)), 1.f));
#pragma unroll
        for (int c = 0; c < 4; ++c)
          if (j >= c && j - c < pitch) tab[c * pitch + j - c] = x;
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = __shfl_sync(0xffffffffu, ctrl->tmem_base, 0);   // provably warp-uniform
  volatile int* abort_flag = &ctrl->abort;

  if (warp == 0) {
    // ---------------------------------------------------------------- TMA producer
    if (lane == 0) {
      mbar_expect_tx(&ctrl->q_full, 2 * kQBytes);
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int h = 0; h < NK; ++h)
          tma_load_3d(q_s + t * kQBytes + h * kHalf, &tmQ, &ctrl->q_full, h * 64, head, q_row0 + t * kQTile);
    }
    __syncwarp();
    const int* table = ROWS ? nullptr : p.block_table + (long long)b * p.max_blocks;
    const int kv_row0 = ROWS ? p.kv_base[b] : 0;
    const int last_page = max((ctx + kPfPage - 1) / kPfPage - 1, 0);
    // Ring items in the order the issuers consume them: K(0), then per KV tile u: K(u+1), V(u).  Q K^T runs one
    // tile ahead of P V, so K(u+2) has the whole of iteration u to arrive.  Item `seq` lives in stage seq % 3.
    int seq = 0;
    bool live = true;
    auto load = [&](bool is_v, int x) {
      if (!live) return;
      const int j = tile_at(x);
      const int st = seq % kKVStages;
      const uint32_t ph = uint32_t(seq / kKVStages) & 1u;
      ++seq;
      bool ok = pf_wait(&ctrl->kv_empty[st], ph ^ 1u, abort_flag, p.status, ERR_WAIT_SMEM_EMPTY);
      if (!__all_sync(0xffffffffu, ok)) { live = false; return; }
      if constexpr (ROWS) {
        if (lane == 0) {
          uint8_t* dst = kv_s + st * kKVBytes;
          const int row = kv_row0 + j * KT;
          mbar_expect_tx(&ctrl->kv_full[st], (is_v ? NV : NK) * kKVHalf);
          if (is_v) {
#pragma unroll
            for (int h = 0; h < NV; ++h) tma_load_3d(dst + h * kKVHalf, &tmV, &ctrl->kv_full[st], h * 64, kvh, row);
          } else {
#pragma unroll
            for (int h = 0; h < NK - 1; ++h) tma_load_3d(dst + h * kKVHalf, &tmK, &ctrl->kv_full[st], h * 64, kvh, row);
            tma_load_2d(dst + (NK - 1) * kKVHalf, &tmR, &ctrl->kv_full[st], 0, row);
          }
        }
      } else {
        constexpr int kPages = KT / kPfPage;
        int blk[kPages];
#pragma unroll
        for (int pi = 0; pi < kPages; ++pi) blk[pi] = table[min(j * kPages + pi, last_page)];
        if (lane == 0) {
          const CUtensorMap* tm = is_v ? &tmV : &tmK;
          uint8_t* dst = kv_s + st * kKVBytes;
          mbar_expect_tx(&ctrl->kv_full[st], kKVBytes);
#pragma unroll
          for (int pi = 0; pi < kPages; ++pi)
#pragma unroll
            for (int h = 0; h < NK; ++h)
              tma_load_4d(dst + h * kKVHalf + pi * (kPfPage * 128), tm, &ctrl->kv_full[st], h * 64, 0, kvh, blk[pi]);
        }
      }
      __syncwarp();
    };
    if (n_union > 0) load(false, 0);
#pragma unroll 1
    for (int u = 0; u < n_union && live; ++u) {
      if (u + 1 < n_union) load(false, u + 1);
      load(true, u);
    }
  } else if (warp == 1 || warp == 2) {
    // ---------------------------------------------------------------- MMA issuers, one per query tile
    // Both issuers walk all KV tiles of the CTA in the producer's order and release every ring stage (the barrier
    // counts two arrivals), also for KV tiles their query tile does not attend to; each waits for a stage to be
    // loaded before it releases it, so that an issuer can never arrive twice on one barrier phase.
    constexpr uint32_t idesc_qk = make_idesc_bf16(128, kKVTile, 0, 0);
    constexpr uint32_t idesc_pv = make_idesc_bf16(128, D, 0, 1);  // B = V is MN-major
    const int t = warp - 1;
    const uint32_t q_lo = uint32_t(make_smem_desc_sw128(smem_u32(q_s + t * kQBytes), 0, 1024));
    const uint32_t kv_lo = uint32_t(make_smem_desc_sw128(smem_u32(kv_s), 0, 1024));
    const uint32_t p_lo = uint32_t(make_smem_desc_sw128(smem_u32(p_s + t * kPBytes), 0, 1024));
    const uint64_t hk = uint64_t(uint32_t(make_smem_desc_sw128(0, 0, 1024) >> 32)) << 32;   // SBO, version, swizzle
    const uint32_t lbo_v = (uint32_t(kKVHalf) >> 4) << 16;                                  // low-word part of V's LBO
    // walk positions of this query tile: the kept tiles and [a_lo, a_hi)
    const int a_lo = kept + (t == 0 ? tr0.lo - u_lo : (two ? tr1.lo - u_lo : 0));
    const int a_hi = kept + (t == 0 ? tr0.hi - u_lo : (two ? tr1.hi - u_lo : 0));
    const auto attends = [&](int x) { return (MODS && x < kept) || (x >= a_lo && x < a_hi); };
    const auto turn_of = [&](int x) { return uint32_t(MODS && x < kept ? x : x - a_lo + kept); };
    const uint32_t s_tmem = tmem_base + kSCol + t * 128, o_tmem = tmem_base + kOCol + t * 128;
    if ((t == 0 || two) && elect_one()) {
      bool ok = pf_wait(&ctrl->q_full, 0, abort_flag, p.status, ERR_WAIT_SMEM_FULL);
      int seq = 0;                                   // ring item counter, in the producer's order
      // K tile x: S_t = Q_t K(x)^T if this query tile attends to it, then release its ring stage
      auto do_k = [&](int x) {
        if (x >= n_union || !ok) return;
        const int item = seq++, st = item % kKVStages;
        ok = pf_wait(&ctrl->kv_full[st], uint32_t(item / kKVStages) & 1u, abort_flag, p.status, ERR_WAIT_SMEM_FULL);
        if (!ok) return;
        if (attends(x)) {
          const uint32_t lit = turn_of(x);
          ok = pf_wait(&ctrl->s_empty[t], (lit & 1u) ^ 1u, abort_flag, p.status, ERR_WAIT_TMEM_EMPTY);
          if (!ok) return;
          tc_fence_after();
          const uint32_t kvd = kv_lo + uint32_t(st * kKVBytes >> 4);
#pragma unroll
          for (int h = 0; h < NK; ++h) {
            uint64_t da[4], db[4];
#pragma unroll
            for (int k4 = 0; k4 < 4; ++k4) {
              da[k4] = hk | (q_lo + uint32_t(h * (kHalf >> 4) + k4 * 2));
              db[k4] = hk | (kvd + uint32_t(h * (kKVHalf >> 4) + k4 * 2));
            }
            umma4_ss(s_tmem, da, db, idesc_qk, h > 0 ? 1u : 0u);
          }
          umma_commit(&ctrl->s_full[t]);
        }
        umma_commit(&ctrl->kv_empty[st]);
      };
      // V tile x: O_t (+)= P_t V(x) if this query tile attends to it, then release its ring stage
      auto do_v = [&](int x) {
        if (!ok) return;
        const int item = seq++, st = item % kKVStages;
        ok = pf_wait(&ctrl->kv_full[st], uint32_t(item / kKVStages) & 1u, abort_flag, p.status, ERR_WAIT_SMEM_FULL);
        if (!ok) return;
        if (attends(x)) {
          const uint32_t lit = turn_of(x);
          ok = pf_wait(&ctrl->p_full[t], lit & 1u, abort_flag, p.status, ERR_WAIT_SOFTMAX);
          if (!ok) return;
          tc_fence_after();
          const uint32_t kvd = kv_lo + uint32_t(st * kKVBytes >> 4);
#pragma unroll
          for (int h = 0; h < KT / 64; ++h) {
            uint64_t da[4], db[4];
#pragma unroll
            for (int k4 = 0; k4 < 4; ++k4) {
              // V tile: [token][64 dims] rows of 128 B; 16 tokens per step = 2 KB; next 64 dims one slab on
              db[k4] = hk | ((kvd + uint32_t((h * 4 + k4) * 128)) | lbo_v);
              da[k4] = hk | (p_lo + uint32_t(h * (kHalf >> 4) + k4 * 2));
            }
            umma4_ss(o_tmem, da, db, idesc_pv, (lit > 0 || h > 0) ? 1u : 0u);
          }
          umma_commit(&ctrl->o_full[t]);            // P_t has been read, O_t holds its product
        }
        umma_commit(&ctrl->kv_empty[st]);
      };
      do_k(0);
#pragma unroll 1
      for (int u = 0; u < n_union && ok; ++u) {
        do_k(u + 1);
        do_v(u);
      }
    }
    __syncwarp();
  } else if (warp >= 4) {
    // ---------------------------------------------------------------- softmax
    const int t = (warp - 4) >> 2;                  // query tile of this warp
    const int quad = warp & 3;                      // TMEM lanes this warp may touch
    const TileRange tr = t == 0 ? tr0 : tr1;
    const int r = quad * 32 + lane;                 // row of the query tile
    const int q_pos = tr.pos0 + r;
    const uint32_t lane_off = uint32_t(quad * 32) << 16;
    const uint32_t s_addr = tmem_base + lane_off + kSCol + t * 128;
    const uint32_t o_addr = tmem_base + lane_off + kOCol + t * 128;
    uint8_t* my_p = p_s + t * kPBytes + r * 128;
    const int n_tiles = (tr.rows > 0 ? kept : 0) + tr.hi - tr.lo;
    // KV tiles of the other query tile
    const int n_other = t == 0 ? (two ? kept + tr1.hi - tr1.lo : 0) : kept + tr0.hi - tr0.lo;
    float m = -INFINITY, l = 0.f;
    int hi_pos = ctx - 1;
    if (p.causal) hi_pos = min(hi_pos, q_pos);
    const int lo_pos = nkb_first_visible(q_pos, p.window, p.chunk);
    bool alive = true;
    constexpr float kLog2e = 1.4426950408889634f;
    const bool capped = MODS && p.mods.softcap > 0.f, distant = MODS && p.mods.dist_a != nullptr;
    const float k_y = capped ? p.scale_log2 / (kLog2e * p.mods.softcap) : 0.f;   // raw score -> argument of tanh
    const float cap2 = p.mods.softcap * kLog2e;
    // the polynomial's coefficients take the scales in (which must not underflow)
    const float poly_raw = capped && fabsf(k_y) > 1e-4f ? 0.35f / fabsf(k_y) : -1.f;
    const float wide_raw = capped ? 1.1f / fmaxf(fabsf(k_y), 1e-30f) : 0.f;
    const float k2 = k_y * k_y, c0 = 0.999999965517f * cap2 * k_y, c1 = -0.333324263276f * cap2 * k_y * k2;
    const float c2 = 0.132958838057f * cap2 * k_y * k2 * k2, c3 = -0.048962819976f * cap2 * k_y * k2 * k2 * k2;
    const int far = MODS ? p.dist_far : 0, first_j = far - q_pos;        // table element of key 0
    const float* dist_row = nullptr;
    if (MODS && far > 0) {
      const int copy = first_j & 3;                                       // tiles start at multiples of four
      dist_row = reinterpret_cast<const float*>(ctrl + 1) + copy * L::pitch_of(far) + (first_j - copy);
    }
    const float dist_a = distant ? p.mods.dist_a[head] : 0.f, dist_b = distant ? p.mods.dist_b[head] : 0.f;
    // raw scores become exponents of two in the exponential's multiply-add, or (MODS) before it
    const float to_log2 = MODS ? 1.f : p.scale_log2;

    for (int it = 0; it < n_tiles; ++it) {
      const int kv0 = (MODS && it < kept ? it : tr.lo + it - kept) * kKVTile;
      bool ok = pf_wait(&ctrl->s_full[t], uint32_t(it) & 1u, abort_flag, p.status, ERR_WAIT_TMEM_FULL);
      if (!__all_sync(0xffffffffu, ok)) { alive = false; break; }
      tc_fence_after();
      uint32_t v[kKVTile];
#pragma unroll
      for (int c = 0; c < kKVTile / 32; ++c) tmem_ld_32x32(s_addr + c * 32, reinterpret_cast<uint32_t(&)[32]>(v[c * 32]));
      tmem_ld_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&ctrl->s_empty[t]);   // the scores are in registers: S_t may be overwritten

      if constexpr (MODS) {
        if (capped) {
          float am4[4];
#pragma unroll
          for (int i = 0; i < 4; ++i) am4[i] = fmaxf(fabsf(__uint_as_float(v[2 * i])), fabsf(__uint_as_float(v[2 * i + 1])));
#pragma unroll
          for (int i = 8; i < kKVTile; i += 2)
            am4[(i >> 1) & 3] = fmax3(am4[(i >> 1) & 3], fabsf(__uint_as_float(v[i])), fabsf(__uint_as_float(v[i + 1])));
          const float am = fmaxf(fmaxf(am4[0], am4[1]), fmaxf(am4[2], am4[3]));
          if (__all_sync(0xffffffffu, am <= poly_raw)) {
            const float2 d0 = make_float2(c0, c0), d1 = make_float2(c1, c1), d2 = make_float2(c2, c2), d3 = make_float2(c3, c3);
#pragma unroll
            for (int i = 0; i < kKVTile; i += 2) {
              const float2 y = make_float2(__uint_as_float(v[i]), __uint_as_float(v[i + 1])), u = fmul2(y, y);
              const float2 w = fmul2(y, ffma2(ffma2(ffma2(u, d3, d2), u, d1), u, d0));
              v[i] = __float_as_uint(w.x);
              v[i + 1] = __float_as_uint(w.y);
            }
          } else if (__all_sync(0xffffffffu, am <= wide_raw)) {
            const float2 ky2 = make_float2(k_y, k_y), cc = make_float2(cap2, cap2);
            const auto dup = [](float x) { return make_float2(x, x); };
#pragma unroll
            for (int i = 0; i < kKVTile; i += 2) {
              const float2 y = fmul2(make_float2(__uint_as_float(v[i]), __uint_as_float(v[i + 1])), ky2), u = fmul2(y, y);
              float2 q = ffma2(u, dup(-0.000275233992f), dup(0.002002967295f));
              q = ffma2(q, u, dup(-0.007526384788f));
              q = ffma2(q, u, dup(0.021194377645f));
              q = ffma2(q, u, dup(-0.053775426680f));
              q = ffma2(q, u, dup(0.133305659147f));
              q = ffma2(q, u, dup(-0.333331798889f));
              q = ffma2(q, u, dup(0.999999985913f));
              const float2 w = fmul2(fmul2(y, cc), q);
              v[i] = __float_as_uint(w.x);
              v[i + 1] = __float_as_uint(w.y);
            }
          } else {
            const float k_e = 2.f * kLog2e * k_y;
#pragma unroll
            for (int i = 0; i < kKVTile; ++i) {
              const float e = exp2f(__uint_as_float(v[i]) * k_e);
              v[i] = __float_as_uint(fmaf(-2.f * cap2, __fdividef(1.f, e + 1.f), cap2));
            }
          }
        } else {
#pragma unroll
          for (int i = 0; i < kKVTile; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * p.scale_log2);
        }
        if (dist_row && it >= kept) {
#pragma unroll
          for (int i = 0; i < kKVTile; i += 4) {
            const float4 d = *reinterpret_cast<const float4*>(dist_row + kv0 + i);
            const float2 a = fadd2(make_float2(__uint_as_float(v[i]), __uint_as_float(v[i + 1])), make_float2(d.x, d.y));
            const float2 b = fadd2(make_float2(__uint_as_float(v[i + 2]), __uint_as_float(v[i + 3])), make_float2(d.z, d.w));
            v[i] = __float_as_uint(a.x);
            v[i + 1] = __float_as_uint(a.y);
            v[i + 2] = __float_as_uint(b.x);
            v[i + 3] = __float_as_uint(b.y);
          }
        } else if (distant) {
          // dist_a ln(1 + dist_b d) in units of ln 2; keys after the query (negative distances) are masked below
          const float d0 = fmaf(dist_b, float(q_pos - kv0), 1.f);
#pragma unroll
          for (int i = 0; i < kKVTile; ++i)
            v[i] = __float_as_uint(fmaf(-dist_a, __log2f(fmaf(-dist_b, float(i), d0)), __uint_as_float(v[i])));
        }
      }
      // the mask only on tiles that cross the causal diagonal, the end of the context or the window edge
      const bool edge = kv0 + kKVTile - 1 > hi_pos || (kv0 < lo_pos && (!MODS || kv0 + kKVTile > p.mods.keep_first));
      if (__any_sync(0xffffffffu, edge)) {
        const int hi_rel = hi_pos - kv0, lo_rel = lo_pos - kv0, keep_rel = MODS ? p.mods.keep_first - kv0 : 0;
#pragma unroll
        for (int i = 0; i < kKVTile; ++i)
          if (i > hi_rel || (i < lo_rel && (!MODS || i >= keep_rel))) v[i] = 0xff800000u;   // -inf
      }
      // four independent chains of three-input maxima instead of one 128-long dependent chain
      float mx4[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) mx4[i] = fmaxf(__uint_as_float(v[2 * i]), __uint_as_float(v[2 * i + 1]));
#pragma unroll
      for (int i = 8; i < kKVTile; i += 2)
        mx4[(i >> 1) & 3] = fmax3(mx4[(i >> 1) & 3], __uint_as_float(v[i]), __uint_as_float(v[i + 1]));
      float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      mx *= to_log2;

      bool p_free = it == 0;     // the P_t buffer may be overwritten (P V of the previous tile has finished)
      if (it == 0) {
        m = mx;
      } else {
        const bool grow = mx > m + kRescaleStep || (m == -INFINITY && mx > -INFINITY);
        if (__any_sync(0xffffffffu, grow)) {
          // O_t holds all of the previous tile's contribution
          ok = pf_wait(&ctrl->o_full[t], uint32_t(it - 1) & 1u, abort_flag, p.status, ERR_WAIT_TMEM_FULL);
          if (!__all_sync(0xffffffffu, ok)) { alive = false; break; }
          p_free = true;
          tc_fence_after();
          const float alpha = grow ? exp2f(m - mx) : 1.f;
#pragma unroll 1
          for (int c = 0; c < D / 32; ++c) {
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
      const float2 sc2 = make_float2(to_log2, to_log2), nb2 = make_float2(-base, -base);
      float2 sum2[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) sum2[i] = make_float2(0.f, 0.f);
      // probabilities of 32 scores as 16 packed bf16 pairs
      auto exp_chunk = [&](int c32, uint32_t (&pk)[16]) {
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const int k = c32 * 32 + 2 * i;
          const float2 x = ffma2(make_float2(__uint_as_float(v[k]), __uint_as_float(v[k + 1])), sc2, nb2);
          const float2 e = make_float2(exp2f(x.x), exp2f(x.y));
          sum2[i & 3] = fadd2(sum2[i & 3], e);
          pk[i] = pack_bf16x2(e.x, e.y);
        }
      };
      // 32 tokens = four 16-byte chunks of the row, swizzled like a TMA 128-byte-swizzle load places them
      auto store_chunk = [&](int c, const uint32_t (&pk)[16]) {
#pragma unroll
        for (int q = 0; q < 4; ++q)
          *reinterpret_cast<uint4*>(my_p + (c >> 1) * kHalf + ((((c & 1) * 4 + q) ^ (r & 7)) << 4)) =
              make_uint4(pk[4 * q], pk[4 * q + 1], pk[4 * q + 2], pk[4 * q + 3]);
      };
      // P_t's buffer is free once P V of the previous tile has finished
      if (!p_free) {
        ok = pf_wait(&ctrl->o_full[t], uint32_t(it - 1) & 1u, abort_flag, p.status, ERR_WAIT_TMEM_FULL);
        if (!__all_sync(0xffffffffu, ok)) { alive = false; break; }
      }
      // The exponentials of the two query tiles take turns.  The warps of tile 0 and tile 1 that own the same TMEM
      // lanes share a scheduler and its special-function unit, which 128 exponentials per row keep busy for about
      // as long as the rest of an iteration takes; left alone the two tiles fall into step (they share the K/V
      // ring), both compute exponentials at half speed and then both wait.  Alternating lets one tile use the unit
      // at full speed while the other loads its scores, takes the maximum and publishes P.
      // Order: tile 0 (it), tile 1 (it), tile 0 (it + 1), ...; a tile that has run out of KV tiles is not waited for.
      if (t == 0 ? (it >= 1 && it - 1 < n_other) : (it < n_other)) {
        ok = pf_wait(&ctrl->turn[t][quad], uint32_t(t == 0 ? it - 1 : it) & 1u, abort_flag, p.status, ERR_WAIT_SOFTMAX);
        if (!__all_sync(0xffffffffu, ok)) { alive = false; break; }
      }
#pragma unroll
      for (int c = 0; c < kKVTile / 32; ++c) {
        uint32_t pk[16];
        exp_chunk(c, pk);
        store_chunk(c, pk);
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
    // ---- epilogue: O_t / l to global memory
    if (tr.rows > 0) {
      bool have_o = false;
      if (alive && n_tiles > 0) {
        bool ok = pf_wait(&ctrl->o_full[t], uint32_t(n_tiles - 1) & 1u, abort_flag, p.status, ERR_WAIT_TMEM_FULL);
        have_o = __all_sync(0xffffffffu, ok);
        if (have_o) tc_fence_after();
      }
      float osc = 1.f;
      if (p.sinks) {
        const float sk = p.sinks[head] * 1.4426950408889634f;
        const float m2 = fmaxf(m, sk);
        osc = (m == -INFINITY) ? 0.f : exp2f(m - m2);
        l = l * osc + exp2f(sk - m2);
      }
      const float inv = l > 0.f ? osc / l : 0.f;
      __nv_bfloat16* dst = p.out + ((long long)(q_row0 + t * kQTile + r) * p.nq + head) * D;
      const bool store = r < tr.rows && !*abort_flag;
#pragma unroll 1
      for (int c = 0; c < D / 32; ++c) {
        uint32_t o[32];
        if (have_o) {
          tmem_ld_32x32(o_addr + c * 32, o);
          tmem_ld_wait();
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i) o[i] = 0u;
        }
        if (store) {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            uint4 w;
            w.x = pack_bf16x2(__uint_as_float(o[i]) * inv, __uint_as_float(o[i + 1]) * inv);
            w.y = pack_bf16x2(__uint_as_float(o[i + 2]) * inv, __uint_as_float(o[i + 3]) * inv);
            w.z = pack_bf16x2(__uint_as_float(o[i + 4]) * inv, __uint_as_float(o[i + 5]) * inv);
            w.w = pack_bf16x2(__uint_as_float(o[i + 6]) * inv, __uint_as_float(o[i + 7]) * inv);
            *reinterpret_cast<uint4*>(dst + c * 32 + i) = w;
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

template <int NK, int NV, int KT, bool ROWS, bool MODS = false>
static int launch_prefill(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const CUtensorMap& tr,
                          PrefillParams p, int batch, int max_q_len, cudaStream_t s) {
  using L = PrefillSmem<NK, NV, KT>;
  constexpr int most = 232448;
  static_assert(L::kBytes <= most && sizeof(PrefillCtrl) % 16 == 0, "shared memory of a CTA");
  int smem = L::kBytes;
  if (MODS && p.mods.dist_a && p.window > 0 && p.window <= 4096) {
    const int far = L::far_of(p.window), bytes = smem + 16 * L::pitch_of(far);
    if (bytes <= most) {
      p.dist_far = far;
      smem = bytes;
    }
  }
  static bool attr_set[64] = {false};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -1;
  if (!attr_set[dev]) {
    cudaError_t e = cudaFuncSetAttribute(flash_attn_prefill_kernel<NK, NV, KT, ROWS, MODS>,
                                         cudaFuncAttributeMaxDynamicSharedMemorySize, MODS ? most : smem);
    if (e != cudaSuccess) return int(e);
    attr_set[dev] = true;
  }
  dim3 grid((max_q_len + kQPair - 1) / kQPair, p.nq, batch);
  return launch_pdl(flash_attn_prefill_kernel<NK, NV, KT, ROWS, MODS>, grid, dim3(kPfThreads), size_t(smem), s, tq, tk, tv, tr, p);
}

}  // namespace nkb

using namespace nkb;

extern "C" int nkb_flash_attn_prefill(const void* q, const void* k_cache, const void* v_cache, const int* block_table,
                                      const int* q_start, const int* q_lens, const int* context_lens, void* out,
                                      int batch, int total_q, int max_q_len, int nq, int nkv, int head_dim,
                                      int block_size, int num_blocks, int max_blocks_per_seq, float scale, int causal,
                                      int window, int chunk, const float* sinks, const NkbScoreMods* mods, void* stream) {
  if (batch <= 0 || total_q <= 0) return 0;
  if (block_size != kPfPage || nq % nkv != 0) return -2;
  if (mods && (mods->keep_first < 0 || (mods->keep_first > 0 && chunk > 0) || !mods->dist_a != !mods->dist_b || (!causal && mods->dist_a)))
    return -2;
  if (!status_word() && nkb_init() != 0) return -1;
  PrefillParams p{};
  p.block_table = block_table;
  p.q_start = q_start;
  p.q_lens = q_lens;
  p.context_lens = context_lens;
  p.out = reinterpret_cast<__nv_bfloat16*>(out);
  p.sinks = sinks;
  p.status = status_word();
  p.nq = nq; p.nkv = nkv; p.max_blocks = max_blocks_per_seq; p.causal = causal; p.window = window; p.chunk = chunk;
  p.scale_log2 = scale * 1.4426950408889634f;
  CUtensorMap tq, tk, tv;
  {
    const uint64_t dims[3] = {uint64_t(head_dim), uint64_t(nq), uint64_t(total_q)};
    const uint64_t strides[2] = {uint64_t(head_dim) * 2, uint64_t(head_dim) * nq * 2};
    const uint32_t box[3] = {64, 1, uint32_t(kQTile)};
    if (encode_tmap_bf16(&tq, q, 3, dims, strides, box)) return -4;
  }
  {
    const uint64_t dims[4] = {uint64_t(head_dim), uint64_t(kPfPage), uint64_t(nkv), uint64_t(num_blocks)};
    const uint64_t strides[3] = {uint64_t(head_dim) * 2, uint64_t(head_dim) * kPfPage * 2,
                                 uint64_t(head_dim) * kPfPage * nkv * 2};
    const uint32_t box[4] = {64, uint32_t(kPfPage), 1, 1};
    if (encode_tmap_bf16(&tk, k_cache, 4, dims, strides, box)) return -4;
    if (encode_tmap_bf16(&tv, v_cache, 4, dims, strides, box)) return -4;
  }
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (mods) {
    p.mods = *mods;
    // tiles of 64 tokens: fewer scores in registers at once, and room for the table beside heads of 128
    if (head_dim == 128) return launch_prefill<2, 2, 64, false, true>(tq, tk, tv, tk, p, batch, max_q_len, s);
    if (head_dim == 64) return launch_prefill<1, 1, 128, false, true>(tq, tk, tv, tk, p, batch, max_q_len, s);
    return -2;
  }
  if (head_dim == 128) return launch_prefill<2, 2, 128, false>(tq, tk, tv, tk, p, batch, max_q_len, s);
  if (head_dim == 64) return launch_prefill<1, 1, 128, false>(tq, tk, tv, tk, p, batch, max_q_len, s);
  return -2;
}

// Prefill attention over expanded latents: kv [rows, ld] holds every head's unrotated key (dim columns each) and then every
// head's value (vdim columns each), rotated [rows, rot_ld] the key part all heads share; position j of sequence b is row
// kv_base[b] + j.  q [total_q, heads, 64 nk] has a head's unrotated part in its first columns and the rotated one in its
// last 64, zeros elsewhere; out is [total_q, heads, 64 nv].  Returns -5 for sizes it does not take.
extern "C" int nkb_latent_prefill(const void* q, const void* kv, const void* rotated, const int* q_start, const int* q_lens,
                                  const int* context_lens, const int* kv_base, void* out, int batch, int total_q, int max_q_len,
                                  int rows, int heads, int dim, int rot, int vdim, long long ld, long long rot_ld, int nk, int nv,
                                  float scale, int window, const float* sinks, void* stream) {
  if (batch <= 0 || total_q <= 0) return 0;
  if (dim < 1 || rot < 1 || vdim < 1 || dim > 64 * (nk - 1) || rot > 64 || vdim > 64 * nv || ((dim | vdim) & 7) || (ld & 7) ||
      (rot_ld & 7) || rot_ld < rot || heads > 65535 || batch > 65535)
    return -5;
  if (rows < 1 || ld < (long long)heads * (dim + vdim)) return -2;
  if (!status_word() && nkb_init() != 0) return -1;
  PrefillParams p{};
  p.q_start = q_start; p.q_lens = q_lens; p.context_lens = context_lens; p.kv_base = kv_base;
  p.out = reinterpret_cast<__nv_bfloat16*>(out);
  p.sinks = sinks;
  p.status = status_word();
  p.nq = heads; p.nkv = heads; p.causal = 1; p.window = window;
  p.scale_log2 = scale * 1.4426950408889634f;
  const int kt = nk == 3 ? 64 : 128;
  CUtensorMap tq, tk, tv, tr;
  {
    const uint64_t dims[3] = {uint64_t(nk) * 64, uint64_t(heads), uint64_t(total_q)};
    const uint64_t strides[2] = {uint64_t(nk) * 128, uint64_t(nk) * 128 * heads};
    const uint32_t box[3] = {64, 1, uint32_t(kQTile)};
    if (encode_tmap_bf16(&tq, q, 3, dims, strides, box)) return -4;
  }
  const auto heads_map = [&](CUtensorMap* m, const void* base, int width) {
    const uint64_t dims[3] = {uint64_t(width), uint64_t(heads), uint64_t(rows)};
    const uint64_t strides[2] = {uint64_t(width) * 2, uint64_t(ld) * 2};
    const uint32_t box[3] = {64, 1, uint32_t(kt)};
    return encode_tmap_bf16(m, base, 3, dims, strides, box);
  };
  if (heads_map(&tk, kv, dim) || heads_map(&tv, reinterpret_cast<const __nv_bfloat16*>(kv) + (long long)heads * dim, vdim)) return -4;
  if (encode_tmap_bf16_2d(&tr, rotated, rot, rows, rot_ld, 64, kt)) return -4;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (nk == 2 && nv == 1) return launch_prefill<2, 1, 128, true>(tq, tk, tv, tr, p, batch, max_q_len, s);
  if (nk == 2 && nv == 2) return launch_prefill<2, 2, 128, true>(tq, tk, tv, tr, p, batch, max_q_len, s);
  if (nk == 3 && nv == 2) return launch_prefill<3, 2, 64, true>(tq, tk, tv, tr, p, batch, max_q_len, s);
  return -5;
}
