// Recurrences with one decay per head and a short convolution in front of them (head_recurrence.h): the gated delta rule and the
// state-space form with a scalar decay.
//
//   conv       y = silu(causal convolution) of all channels of packed prompts; a second launch leaves the last inputs of every
//              sequence in its slot (the first one still reads what earlier steps left there)
//   scan       any number of new tokens per sequence.  A CTA owns some columns of one head of one sequence for all of its
//              tokens; eight lanes share NC columns, each holding every eighth group of four channels of them in registers.
//              Both S^T k and S^T q are taken from the state before its update, since after it
//                  S^T q = g (S_old^T q) + (k . q) u,
//              so a token needs one exchange of sums between lanes: a transposing butterfly over the 2 NC sums.  Unit norms,
//              scales and step sizes are factors of these sums, folded into five numbers per token.  A tile of tokens is copied
//              as it is while the previous one is multiplied.
//   step       one new token per sequence (decode).  A CTA owns a head of a sequence, streams its state through registers once
//              and computes everything around it itself: the convolution of its channels, unit norms, decay, step size, and
//              (per-head norms) the norm and gate of the result.
//   group norm out = norm_w * x / sqrt(mean over the element's part of x^2 + eps), x = y * gate_act(g): results whose norm spans
//              heads and follows the gate
//
// State arithmetic is fp32 throughout.
#include "common.cuh"
#include "proj_src.cuh"
#include "activations.cuh"
#include "head_recurrence.h"
#include "api.h"

namespace nkb {

__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// ------------------------------------------------------------------------------------------------ convolution
struct ShortConvParams {
  NkbProj x;
  const float *w, *b;
  float* state;
  const int *slot_ids, *q_start, *q_lens, *context_lens;
  void* out;                // [tokens, channels]
  int batch, tokens, channels, taps, act, run;      // run: tokens of a CTA
};
constexpr int kConvTokens = 64;     // at most
constexpr int kMaxTaps = 8;

// V channels of a row: as they lie in memory (bf16 in one piece), and as numbers
template <int V>
struct ChanRaw {
  float x;
  __device__ __forceinline__ void load(const NkbProj& s, long long row, int c) { x = proj_load(s, row, c); }
  __device__ __forceinline__ void get(float (&o)[V]) const { o[0] = x; }
};
template <>
struct ChanRaw<4> {
  uint2 r;
  __device__ __forceinline__ void load(const NkbProj& s, long long row, int c) {
    r = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(s.ptr) + row * s.ld + c);
  }
  __device__ __forceinline__ void get(float (&o)[4]) const {
    const float2 a = unpack_bf16x2(r.x), b = unpack_bf16x2(r.y);
    o[0] = a.x; o[1] = a.y; o[2] = b.x; o[3] = b.y;
  }
};
template <>
struct ChanRaw<8> {
  uint4 r;
  __device__ __forceinline__ void load(const NkbProj& s, long long row, int c) {
    r = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(s.ptr) + row * s.ld + c);
  }
  __device__ __forceinline__ void get(float (&o)[8]) const {
    const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 f = unpack_bf16x2(w[e]);
      o[2 * e] = f.x;
      o[2 * e + 1] = f.y;
    }
  }
};

// z sigmoid(z) with the approximate exponential and reciprocal, for results that are stored in bf16
__device__ __forceinline__ float silu_fast(float z) {
  float e, r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(-1.4426950408889634f * z));
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + e));
  return z * r;
}

// A CTA owns a run of tokens and 128 V channels; V = 4: finished bf16 values in aligned pieces of four.  Four tokens are loaded while
// the four before them are computed.  seq_of: the token's sequence.
template <int V, int TAPS, typename OutT>
__global__ void __launch_bounds__(128) short_conv_kernel(const __grid_constant__ ShortConvParams p) {
  constexpr int H = TAPS > 1 ? TAPS - 1 : 1, AHEAD = 4;
  __shared__ int seq_of[kConvTokens];
  const int t0 = blockIdx.y * p.run, nt = min(p.run, p.tokens - t0);
  const int c = (blockIdx.x * 128 + threadIdx.x) * V;
  if (threadIdx.x < kConvTokens) seq_of[threadIdx.x] = -1;
  float w[TAPS][V], bias[V];
  if (c < p.channels) {
#pragma unroll
    for (int e = 0; e < V; ++e) {
      bias[e] = p.b ? p.b[c + e] : 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) w[j][e] = p.w[(long long)j * p.channels + c + e];
    }
  }
  griddep_wait();
  griddep_launch();
  ChanRaw<V> cur[AHEAD], next[AHEAD];
  const auto fetch = [&](ChanRaw<V> (&r)[AHEAD], int i0) {
#pragma unroll
    for (int k = 0; k < AHEAD; ++k) r[k].load(p.x, t0 + min(i0 + k, nt - 1), c);
  };
  if (c < p.channels) fetch(cur, 0);
  __syncthreads();
  for (int b = threadIdx.x; b < p.batch; b += 128) {
    const int s = p.q_start[b], e = s + p.q_lens[b];
    for (int t = max(s, t0); t < min(e, t0 + nt); ++t) seq_of[t - t0] = b;
  }
  __syncthreads();
  if (c >= p.channels) return;
  OutT* out = reinterpret_cast<OutT*>(p.out);
  float past[H][V];                                  // past[l]: input of the token l + 1 before the current one
#pragma unroll
  for (int l = 0; l < H; ++l)
#pragma unroll
    for (int e = 0; e < V; ++e) past[l][e] = 0.f;
  int seq = -1;
#pragma unroll 1
  for (int i0 = 0; i0 < nt; i0 += AHEAD) {
    fetch(next, i0 + AHEAD);                         // (past the end: the last token again)
#pragma unroll
    for (int k = 0; k < AHEAD; ++k) {
      const int i = i0 + k;
      if (i >= nt) break;
      const long long t = t0 + i;
      float x[V];
      cur[k].get(x);
      const int b = seq_of[i];
      if (b >= 0 && b != seq) {                      // what precedes the first of this CTA's tokens of the sequence
        const int first = p.q_start[b], n = p.q_lens[b], ctx = p.context_lens[b];
        const float* st = p.state + (long long)(p.slot_ids ? p.slot_ids[b] : b) * TAPS * p.channels + c;
#pragma unroll
        for (int l = 0; l < TAPS - 1; ++l) {
          const long long from = t - 1 - l;
          const int pos = ctx - n + int(from - first);
          if (from >= first) {
            ChanRaw<V> r;
            r.load(p.x, from, c);
            r.get(past[l]);
          } else {
#pragma unroll
            for (int e = 0; e < V; ++e) past[l][e] = ctx >= n && pos >= 0 ? st[(long long)(pos % TAPS) * p.channels + e] : 0.f;
          }
        }
      }
      seq = b;
      float y[V];
#pragma unroll
      for (int e = 0; e < V; ++e) {
        y[e] = fmaf(w[TAPS - 1][e], x[e], bias[e]);
#pragma unroll
        for (int l = 0; l < TAPS - 1; ++l) y[e] = fmaf(w[TAPS - 2 - l][e], past[l][e], y[e]);
      }
      if (sizeof(OutT) == 2 && p.act == ACT_SILU) {
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] = silu_fast(y[e]);
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] = apply_act(y[e], p.act);
      }
      OutT* o = out + t * p.channels + c;
      if constexpr (V == 4) {
        *reinterpret_cast<uint2*>(o) = make_uint2(pack_bf16x2(y[0], y[1]), pack_bf16x2(y[2], y[3]));
      } else {
        o[0] = cast_out<OutT>(y[0]);
      }
#pragma unroll
      for (int l = TAPS - 2; l > 0; --l)
#pragma unroll
        for (int e = 0; e < V; ++e) past[l][e] = past[l - 1][e];
      if constexpr (TAPS > 1) {
#pragma unroll
        for (int e = 0; e < V; ++e) past[0][e] = x[e];
      }
    }
#pragma unroll
    for (int k = 0; k < AHEAD; ++k) cur[k] = next[k];
  }
}

// Inputs of the last tokens (at most taps of them) of every sequence into its slot.
__global__ void __launch_bounds__(256) conv_state_kernel(const __grid_constant__ ShortConvParams p) {
  const int c = blockIdx.x * 256 + threadIdx.x, b = blockIdx.y;
  griddep_wait();
  griddep_launch();
  const int n = p.q_lens[b], ctx = p.context_lens[b];
  if (c >= p.channels || n <= 0 || ctx < n) return;
  float* st = p.state + (long long)(p.slot_ids ? p.slot_ids[b] : b) * p.taps * p.channels + c;
  for (int j = 0; j < min(n, p.taps); ++j)
    st[(long long)((ctx - 1 - j) % p.taps) * p.channels] = proj_load(p.x, p.q_start[b] + n - 1 - j, c);
}

template <int V, typename OutT>
static int launch_conv(ShortConvParams p, cudaStream_t s) {
  // long runs (what precedes a run is read again), as long as the grid fills the device a few times over
  const int cols = (p.channels + 128 * V - 1) / (128 * V);
  p.run = kConvTokens;
  while (p.run > 4 && (long long)cols * ((p.tokens + p.run - 1) / p.run) < 148 * 16) p.run /= 2;
  const dim3 grid(cols, (p.tokens + p.run - 1) / p.run), block(128);
  switch (p.taps) {
    case 1: return launch_pdl(short_conv_kernel<V, 1, OutT>, grid, block, 0, s, p);
    case 2: return launch_pdl(short_conv_kernel<V, 2, OutT>, grid, block, 0, s, p);
    case 3: return launch_pdl(short_conv_kernel<V, 3, OutT>, grid, block, 0, s, p);
    case 4: return launch_pdl(short_conv_kernel<V, 4, OutT>, grid, block, 0, s, p);
    case 5: return launch_pdl(short_conv_kernel<V, 5, OutT>, grid, block, 0, s, p);
    case 6: return launch_pdl(short_conv_kernel<V, 6, OutT>, grid, block, 0, s, p);
    case 7: return launch_pdl(short_conv_kernel<V, 7, OutT>, grid, block, 0, s, p);
    case 8: return launch_pdl(short_conv_kernel<V, 8, OutT>, grid, block, 0, s, p);
  }
  return -2;
}

// ------------------------------------------------------------------------------------------------ scan
constexpr int kRecThreads = 128;
constexpr int kRecLanes = 8;       // lanes that share a set of columns

__device__ __forceinline__ void rec_cp16(void* dst, const void* src, bool on) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(on ? 16 : 0) : "memory");
}

template <int CL, int NC>
struct RecShape {
  static constexpr int TT = CL <= 16 ? 16 : 8;              // tokens per tile
  static constexpr int DP = kRecLanes * CL, COLS = 16 * NC;
  static constexpr int kWork = TT * (2 * DP + 2 * COLS) * 4;    // fp32 queries, keys, values, results
  static constexpr int kRaw = TT * (2 * DP + COLS) * 2;         // bf16 queries, keys, values
};

// The five factors of a token (see the head of the file): u' = (factor of k) u is what the update multiplies with raw keys.
struct __align__(16) RecFactors {
  float g, ev, es, oq, ou;   // S <- g S + k u';  u' = ev v - es (S^T k);  o = oq (S^T q) + ou u'
  float pad[3];
};

// CL: channels per lane (dim <= 8 CL), NC: columns per lane group.  ASYNC: bf16 rows in aligned runs of eight channels.
template <int CL, int NC, bool DELTA, bool ASYNC, typename OutT>
__global__ void __launch_bounds__(kRecThreads, CL <= 16 ? 4 : 2) head_rec_scan_kernel(const __grid_constant__ NkbHeadRec p) {
  using S = RecShape<CL, NC>;
  constexpr int TT = S::TT, DP = S::DP, COLS = S::COLS;
  constexpr int QW = DP / 4;                        // threads that prepare one token's channels
  constexpr int RW = QW < 32 ? QW : 32, BW = QW / RW;
  constexpr int SUMS = DELTA ? 2 * NC : kRecLanes;  // sums of an exchange
  constexpr int TB = DELTA ? 1 : kRecLanes / NC;    // tokens whose sums are exchanged together
  constexpr int REP = kRecLanes / SUMS;             // lanes that end up with the same sum
  extern __shared__ __align__(16) uint8_t rec_s[];
  float(*qs)[DP] = reinterpret_cast<float(*)[DP]>(rec_s);
  float(*ks)[DP] = qs + TT;
  float(*vs)[COLS] = reinterpret_cast<float(*)[COLS]>(ks + TT);
  float(*os)[COLS] = vs + TT;
  __nv_bfloat16(*qr)[DP] = reinterpret_cast<__nv_bfloat16(*)[DP]>(os + TT);
  __nv_bfloat16(*kr)[DP] = qr + TT;
  __nv_bfloat16(*vr)[COLS] = reinterpret_cast<__nv_bfloat16(*)[COLS]>(kr + TT);
  __shared__ RecFactors fac[TT];
  __shared__ float dots[TT][BW][3];                 // q.q, k.k, q.k of a token
  const int head = blockIdx.y, b = blockIdx.z, col0 = blockIdx.x * COLS;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane & 7;
  const int cl0 = (warp * 4 + (lane >> 3)) * NC;    // first of this lane's columns within the CTA
  const int kvh = head / (p.heads / p.groups);
  const int hq = p.q_col + kvh * p.dim, hk = p.k_col + kvh * p.dim, hv = p.v_col + head * p.vdim;
  const int dim_p = (p.dim + 3) / 4 * 4, pc = (threadIdx.x % QW) * 4;
  const float rate = p.rate[head], dtb = p.dt_bias[head], skip = p.skip ? p.skip[head] : 0.f;
  griddep_wait();
  griddep_launch();
  const int n = p.q_lens[b], ctx = p.context_lens[b];
  if (n <= 0 || ctx < n) return;
  const long long row0 = p.q_start[b];
  const int slot = p.slot_ids ? p.slot_ids[b] : b;
  const bool fresh = ctx == n;
  float* st = p.state + (((long long)slot * p.heads + head) * p.vdim + col0 + cl0) * dim_p;

  const __nv_bfloat16* xb = reinterpret_cast<const __nv_bfloat16*>(p.x.ptr);
  float a_raw = 0.f, b_raw = 0.f;                   // of token threadIdx.x of the tile that is on its way
  auto fetch = [&](int t0) {
    if constexpr (ASYNC) {
#pragma unroll
      for (int i = 0; i < (TT * DP / 8 + kRecThreads - 1) / kRecThreads; ++i) {
        const int idx = threadIdx.x + i * kRecThreads, tok = idx / (DP / 8), c = idx % (DP / 8) * 8;
        if (idx < TT * DP / 8) {
          const bool on = t0 + tok < n && c < p.dim;
          const __nv_bfloat16* row = xb + (on ? row0 + t0 + tok : row0) * p.x.ld;
          rec_cp16(&qr[tok][c], row + (on ? hq + c : hq), on);
          rec_cp16(&kr[tok][c], row + (on ? hk + c : hk), on);
        }
      }
#pragma unroll
      for (int i = 0; i < (TT * COLS / 8 + kRecThreads - 1) / kRecThreads; ++i) {
        const int idx = threadIdx.x + i * kRecThreads, tok = idx / (COLS / 8), c = idx % (COLS / 8) * 8;
        if (idx < TT * COLS / 8) {
          const bool on = t0 + tok < n && col0 + c < p.vdim;
          rec_cp16(&vr[tok][c], xb + (on ? row0 + t0 + tok : row0) * p.x.ld + hv + (on ? col0 + c : 0), on);
        }
      }
      asm volatile("cp.async.commit_group;" ::: "memory");
    }
    if (threadIdx.x < TT && t0 + int(threadIdx.x) < n) {
      a_raw = proj_load(p.a, row0 + t0 + threadIdx.x, head);
      if (DELTA) b_raw = proj_load(p.b, row0 + t0 + threadIdx.x, head);
    }
  };
  auto prepare = [&](int t0) {
#pragma unroll
    for (int i = 0; i < (TT * QW + kRecThreads - 1) / kRecThreads; ++i) {
      const int idx = threadIdx.x + i * kRecThreads, tok = idx / QW;
      if (TT * QW < kRecThreads && idx >= TT * QW) break;      // whole warps
      const bool on = t0 + tok < n && pc < p.dim;
      float q[4] = {0.f, 0.f, 0.f, 0.f}, k[4] = {0.f, 0.f, 0.f, 0.f};
      if (on) {
        if constexpr (ASYNC) {
          const uint2 qu = *reinterpret_cast<const uint2*>(&qr[tok][pc]), ku = *reinterpret_cast<const uint2*>(&kr[tok][pc]);
          const float2 q0 = unpack_bf16x2(qu.x), q1 = unpack_bf16x2(qu.y), k0 = unpack_bf16x2(ku.x), k1 = unpack_bf16x2(ku.y);
          q[0] = q0.x; q[1] = q0.y; q[2] = q1.x; q[3] = q1.y;
          k[0] = k0.x; k[1] = k0.y; k[2] = k1.x; k[3] = k1.y;
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (pc + e < p.dim) {
              q[e] = proj_load(p.x, row0 + t0 + tok, hq + pc + e);
              k[e] = proj_load(p.x, row0 + t0 + tok, hk + pc + e);
            }
        }
      }
      *reinterpret_cast<float4*>(&qs[tok][pc]) = make_float4(q[0], q[1], q[2], q[3]);
      *reinterpret_cast<float4*>(&ks[tok][pc]) = make_float4(k[0], k[1], k[2], k[3]);
      float qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        qq = fmaf(q[e], q[e], qq);
        kk = fmaf(k[e], k[e], kk);
        qk = fmaf(q[e], k[e], qk);
      }
#pragma unroll
      for (int w = RW / 2; w > 0; w >>= 1) {
        if (DELTA) {
          qq += __shfl_xor_sync(0xffffffffu, qq, w);
          kk += __shfl_xor_sync(0xffffffffu, kk, w);
        }
        qk += __shfl_xor_sync(0xffffffffu, qk, w);
      }
      if ((threadIdx.x & (RW - 1)) == 0) {
        float* d = dots[tok][BW > 1 ? (idx % QW) / 32 : 0];
        d[0] = qq; d[1] = kk; d[2] = qk;
      }
    }
#pragma unroll
    for (int i = 0; i < (TT * COLS + kRecThreads - 1) / kRecThreads; ++i) {
      const int idx = threadIdx.x + i * kRecThreads, tok = idx / COLS, c = idx % COLS;
      if constexpr (ASYNC) {
        vs[tok][c] = __bfloat162float(vr[tok][c]);
      } else {
        vs[tok][c] = t0 + tok < n && col0 + c < p.vdim ? proj_load(p.x, row0 + t0 + tok, hv + col0 + c) : 0.f;
      }
    }
  };
  // tokens past the end keep the state (decay one, nothing written); their results are not stored
  auto factors = [&](int t0) {
    if (threadIdx.x >= TT) return;
    const int i = threadIdx.x;
    RecFactors f{1.f, 0.f, 0.f, 0.f, 0.f, {0.f, 0.f, 0.f}};
    if (t0 + i < n) {
      float qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
      for (int w = 0; w < BW; ++w) {
        qq += dots[i][w][0];
        kk += dots[i][w][1];
        qk += dots[i][w][2];
      }
      const float dt = softplus_f(a_raw + dtb);
      f.g = expf(-rate * dt);
      if (DELTA) {
        const float iq = p.q_scale / sqrtf(qq + p.unit_eps), ik = 1.f / sqrtf(kk + p.unit_eps);
        f.ev = ik / (1.f + expf(-b_raw));
        f.es = f.ev * f.g * ik;
        f.oq = iq * f.g;
        f.ou = iq * qk;
      } else {
        f.ev = dt;
        f.oq = p.q_scale * f.g;
        f.ou = p.q_scale * qk;
      }
    }
    fac[i] = f;
  };
  fetch(0);

  // channels of this lane: groups of four, group j at (j * 8 + g) * 4
  float2 D[NC][CL / 2];
#pragma unroll
  for (int k = 0; k < NC; ++k) {
    const bool ok = col0 + cl0 + k < p.vdim;
#pragma unroll
    for (int j = 0; j < CL / 4; ++j) {
      const int c = (j * kRecLanes + g) * 4;
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!fresh && ok && c < dim_p) x = *reinterpret_cast<const float4*>(st + (long long)k * dim_p + c);
      D[k][2 * j] = make_float2(x.x, x.y);
      D[k][2 * j + 1] = make_float2(x.z, x.w);
    }
  }

#pragma unroll 1
  for (int t0 = 0; t0 < n; t0 += TT) {
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();                                 // the raw tile is there; nobody reads the fp32 tile or os any more
    prepare(t0);
    __syncthreads();
    factors(t0);
    __syncthreads();
    if (t0 + TT < n) fetch(t0 + TT);
#pragma unroll 1
    for (int h = 0; h < TT; h += TB) {
      if (t0 + h >= n) break;
      float po[SUMS];
#pragma unroll
      for (int tt = 0; tt < TB; ++tt) {
        const int tok = h + tt;
        const float4 f4 = *reinterpret_cast<const float4*>(&fac[tok]);       // g, ev, es, oq
        float2 sk[NC], sq[NC];
#pragma unroll
        for (int k = 0; k < NC; ++k) sk[k] = sq[k] = make_float2(0.f, 0.f);
        const float2 g2 = make_float2(f4.x, f4.x);
        if constexpr (DELTA) {
#pragma unroll
          for (int j = 0; j < CL / 4; ++j) {
            const int c = (j * kRecLanes + g) * 4;
            const float4 q4 = *reinterpret_cast<const float4*>(&qs[tok][c]), k4 = *reinterpret_cast<const float4*>(&ks[tok][c]);
            const float2 q2[2] = {make_float2(q4.x, q4.y), make_float2(q4.z, q4.w)};
            const float2 k2[2] = {make_float2(k4.x, k4.y), make_float2(k4.z, k4.w)};
#pragma unroll
            for (int k = 0; k < NC; ++k)
#pragma unroll
              for (int i = 0; i < 2; ++i) {
                sk[k] = ffma2(k2[i], D[k][2 * j + i], sk[k]);
                sq[k] = ffma2(q2[i], D[k][2 * j + i], sq[k]);
              }
          }
#pragma unroll
          for (int k = 0; k < NC; ++k) {
            po[k] = sk[k].x + sk[k].y;
            po[NC + k] = sq[k].x + sq[k].y;
          }
          // eight lanes x SUMS sums: lane g ends with sum g / REP
#pragma unroll
          for (int w = SUMS / 2; w > 0; w >>= 1) {
#pragma unroll
            for (int i = 0; i < w; ++i) {
              const bool up = g & (w * REP);
              const float keep = up ? po[w + i] : po[i], send = up ? po[i] : po[w + i];
              po[i] = keep + __shfl_xor_sync(0xffffffffu, send, w * REP);
            }
          }
#pragma unroll
          for (int w = REP / 2; w > 0; w >>= 1) po[0] += __shfl_xor_sync(0xffffffffu, po[0], w);
          const int mine = g / REP;                                          // < NC: S^T k, otherwise S^T q
          const float u = fmaf(f4.y, vs[tok][cl0 + (mine % NC)], -f4.z * po[0]);
          float2 u2[NC];
#pragma unroll
          for (int k = 0; k < NC; ++k) {
            const float x = __shfl_sync(0xffffffffu, u, (lane & 24) + k * REP);
            u2[k] = make_float2(x, x);
          }
          const float own = __shfl_sync(0xffffffffu, u, (lane & 24) + (mine % NC) * REP);
          if (mine >= NC && g % REP == 0) os[tok][cl0 + mine - NC] = fmaf(f4.w, po[0], fac[tok].ou * own);
#pragma unroll
          for (int j = 0; j < CL / 4; ++j) {
            const float4 k4 = *reinterpret_cast<const float4*>(&ks[tok][(j * kRecLanes + g) * 4]);
            const float2 k2[2] = {make_float2(k4.x, k4.y), make_float2(k4.z, k4.w)};
#pragma unroll
            for (int k = 0; k < NC; ++k)
#pragma unroll
              for (int i = 0; i < 2; ++i) D[k][2 * j + i] = ffma2(k2[i], u2[k], fmul2(g2, D[k][2 * j + i]));
          }
        } else {
          float2 u2[NC];
#pragma unroll
          for (int k = 0; k < NC; ++k) {
            const float x = f4.y * vs[tok][cl0 + k];
            u2[k] = make_float2(x, x);
          }
#pragma unroll
          for (int j = 0; j < CL / 4; ++j) {
            const int c = (j * kRecLanes + g) * 4;
            const float4 q4 = *reinterpret_cast<const float4*>(&qs[tok][c]), k4 = *reinterpret_cast<const float4*>(&ks[tok][c]);
            const float2 q2[2] = {make_float2(q4.x, q4.y), make_float2(q4.z, q4.w)};
            const float2 k2[2] = {make_float2(k4.x, k4.y), make_float2(k4.z, k4.w)};
#pragma unroll
            for (int k = 0; k < NC; ++k)
#pragma unroll
              for (int i = 0; i < 2; ++i) {
                float2& d = D[k][2 * j + i];
                sq[k] = ffma2(q2[i], d, sq[k]);
                d = ffma2(k2[i], u2[k], fmul2(g2, d));
              }
          }
#pragma unroll
          for (int k = 0; k < NC; ++k) po[tt * NC + k] = sq[k].x + sq[k].y;
        }
      }
      if constexpr (!DELTA) {
#pragma unroll
        for (int w = kRecLanes / 2; w > 0; w >>= 1) {
#pragma unroll
          for (int i = 0; i < w; ++i) {
            const float keep = (g & w) ? po[w + i] : po[i], send = (g & w) ? po[i] : po[w + i];
            po[i] = keep + __shfl_xor_sync(0xffffffffu, send, w);
          }
        }
        os[h + g / NC][cl0 + g % NC] = po[0];
      }
    }
    __syncthreads();
    OutT* out = reinterpret_cast<OutT*>(p.out);
#pragma unroll
    for (int i = 0; i < (TT * COLS + kRecThreads - 1) / kRecThreads; ++i) {
      const int idx = threadIdx.x + i * kRecThreads, tok = idx / COLS, c = idx % COLS;
      if (t0 + tok < n && col0 + c < p.vdim) {
        float r = os[tok][c];
        if constexpr (!DELTA) {
          const float v = vs[tok][c];
          r = fmaf(fac[tok].oq, r, fmaf(fac[tok].ou * fac[tok].ev, v, skip * v));
        }
        out[((row0 + t0 + tok) * p.heads + head) * p.vdim + col0 + c] = cast_out<OutT>(r);
      }
    }
  }
#pragma unroll
  for (int k = 0; k < NC; ++k)
#pragma unroll
    for (int j = 0; j < CL / 4; ++j) {
      const int c = (j * kRecLanes + g) * 4;
      if (col0 + cl0 + k < p.vdim && c < dim_p)
        *reinterpret_cast<float4*>(st + (long long)k * dim_p + c) =
            make_float4(D[k][2 * j].x, D[k][2 * j].y, D[k][2 * j + 1].x, D[k][2 * j + 1].y);
    }
}

template <int CL, int NC, bool DELTA, bool ASYNC, typename OutT>
static int launch_rec_one(const NkbHeadRec& p, cudaStream_t s) {
  using S = RecShape<CL, NC>;
  constexpr int smem = S::kWork + (ASYNC ? S::kRaw : 0);
  auto kernel = head_rec_scan_kernel<CL, NC, DELTA, ASYNC, OutT>;
  static bool attr_set[64] = {false};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -1;
  if (!attr_set[dev]) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return int(e);
    attr_set[dev] = true;
  }
  return launch_pdl(kernel, dim3((p.vdim + S::COLS - 1) / S::COLS, p.heads, p.batch), dim3(kRecThreads), size_t(smem), s, p);
}
template <int CL, int NC>
static int launch_rec_form(const NkbHeadRec& p, bool async, cudaStream_t s) {
  using bf = __nv_bfloat16;
  const bool delta = p.b.ptr != nullptr;
  if (async) return delta ? launch_rec_one<CL, NC, true, true, bf>(p, s) : launch_rec_one<CL, NC, false, true, bf>(p, s);
  if (p.bf16) return delta ? launch_rec_one<CL, NC, true, false, bf>(p, s) : launch_rec_one<CL, NC, false, false, bf>(p, s);
  return delta ? launch_rec_one<CL, NC, true, false, float>(p, s) : launch_rec_one<CL, NC, false, false, float>(p, s);
}
// More columns per lane mean fewer shared-memory reads per state element, fewer mean more warps to hide latency with.
template <int CL>
static int launch_rec(const NkbHeadRec& p, bool async, cudaStream_t s) {
  if ((long long)p.batch * p.heads * ((p.vdim + 63) / 64) >= 2 * 148) return launch_rec_form<CL, 4>(p, async, s);
  return launch_rec_form<CL, 2>(p, async, s);
}

// ------------------------------------------------------------------------------------------------ step
constexpr int kRecStepThreads = 256;
constexpr int kRecStepBlocks = 4;   // column blocks of 32 in flight

template <int CH, bool DELTA, typename OutT>
__global__ void __launch_bounds__(kRecStepThreads) head_rec_step_kernel(const __grid_constant__ NkbHeadRec p) {
  constexpr int D8 = 8 * CH;
  __shared__ __align__(16) float qs[D8], ks[D8];
  __shared__ float red[kRecStepThreads / 32], gates[3];      // decay, step size, write strength
  extern __shared__ float dyn[];                    // v, o, norm weight times gate [vdim] each
  float* vs = dyn;
  float* os = dyn + p.vdim;
  float* gs = os + p.vdim;
  const int head = blockIdx.x, b = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane & 7;
  const int cl = warp * 4 + (lane >> 3);
  const int per = p.heads / p.groups, kvh = head / per, hv = head * p.vdim, dim_p = (p.dim + 3) / 4 * 4;
  griddep_wait();
  griddep_launch();
  const bool finish = p.norm_w != nullptr;
  const long long o_row = (long long)b * p.heads * p.vdim + hv;
  auto put = [&](int c, float v) {
    if (finish) reinterpret_cast<OutT*>(p.out)[o_row + c] = cast_out<OutT>(v);
    else reinterpret_cast<float*>(p.out)[o_row + c] = v;
  };
  const int ctx = p.context_lens[b];
  if (ctx <= 0) {
    for (int c = threadIdx.x; c < p.vdim; c += kRecStepThreads) put(c, 0.f);
    return;
  }
  const int slot = p.slot_ids ? p.slot_ids[b] : b, pos = ctx - 1;
  const bool fresh = pos == 0;
  float* st = p.state + ((long long)slot * p.heads + head) * p.vdim * dim_p;
  float* ring = p.conv_state + (long long)slot * p.taps * p.channels;
  // the convolution of one channel; its owner leaves the input in the ring
  auto channel = [&](int c, bool owner) {
    const float x = proj_load(p.x, b, c);
    float y = fmaf(p.conv_w[(long long)(p.taps - 1) * p.channels + c], x, p.conv_b ? p.conv_b[c] : 0.f);
    for (int l = 1; l < p.taps && l <= pos; ++l)
      y = fmaf(p.conv_w[(long long)(p.taps - 1 - l) * p.channels + c], ring[(long long)((pos - l) % p.taps) * p.channels + c], y);
    if (owner) ring[(long long)(pos % p.taps) * p.channels + c] = x;
    return y / (1.f + expf(-y));
  };
  const int nblk = (p.vdim + 31) / 32;
  float g_t = 0.f, ev = 0.f, es = 0.f, oq = 0.f, ou = 0.f;
  for (int b0 = 0; b0 < nblk; b0 += kRecStepBlocks) {
    float4 S[kRecStepBlocks][CH / 4];
#pragma unroll
    for (int k = 0; k < kRecStepBlocks; ++k) {
      const int col = (b0 + k) * 32 + cl;
#pragma unroll
      for (int j = 0; j < CH / 4; ++j) {
        const int c = (j * 8 + g) * 4;
        S[k][j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (!fresh && col < p.vdim && c < dim_p)
          S[k][j] = __ldcs(reinterpret_cast<const float4*>(st + (long long)col * dim_p + c));
      }
    }
    if (b0 == 0) {
      for (int i = threadIdx.x; i < 2 * D8 + p.vdim; i += kRecStepThreads) {
        if (i < 2 * D8) {
          const int c = i < D8 ? i : i - D8;
          const float y = c < p.dim ? channel((i < D8 ? p.q_col : p.k_col) + kvh * p.dim + c, head % per == 0) : 0.f;
          (i < D8 ? qs : ks)[c] = y;
        } else {
          const int c = i - 2 * D8;
          vs[c] = channel(p.v_col + hv + c, true);
          if (finish) gs[c] = p.norm_w[c] * apply_act(proj_load(p.g, b, hv + c), p.gate_act);
        }
      }
      if (threadIdx.x == kRecStepThreads - 1) {
        const float dt = softplus_f(proj_load(p.a, b, head) + p.dt_bias[head]);
        gates[0] = expf(-p.rate[head] * dt);
        gates[1] = dt;
        gates[2] = DELTA ? 1.f / (1.f + expf(-proj_load(p.b, b, head))) : 0.f;
      }
      __syncthreads();
      float qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
      for (int c = lane; c < D8; c += 32) {
        const float q = qs[c], k = ks[c];
        qq = fmaf(q, q, qq);
        kk = fmaf(k, k, kk);
        qk = fmaf(q, k, qk);
      }
      qk = warp_sum(qk);
      g_t = gates[0];
      if constexpr (DELTA) {
        const float iq = p.q_scale / sqrtf(warp_sum(qq) + p.unit_eps), ik = 1.f / sqrtf(warp_sum(kk) + p.unit_eps);
        ev = ik * gates[2];
        es = ev * g_t * ik;
        oq = iq * g_t;
        ou = iq * qk;
      } else {
        ev = gates[1];
        oq = p.q_scale * g_t;
        ou = p.q_scale * qk;
      }
    }
#pragma unroll
    for (int k = 0; k < kRecStepBlocks; ++k) {
      const int col = (b0 + k) * 32 + cl;
      const bool ok = col < p.vdim;
      const float v = ok ? vs[col] : 0.f;
      float sk = 0.f, sq = 0.f;
#pragma unroll
      for (int j = 0; j < CH / 4; ++j) {
        const int c = (j * 8 + g) * 4;
        const float4 q4 = *reinterpret_cast<const float4*>(&qs[c]), s = S[k][j];
        sq = fmaf(q4.x, s.x, sq);
        sq = fmaf(q4.y, s.y, sq);
        sq = fmaf(q4.z, s.z, sq);
        sq = fmaf(q4.w, s.w, sq);
        if constexpr (DELTA) {
          const float4 k4 = *reinterpret_cast<const float4*>(&ks[c]);
          sk = fmaf(k4.x, s.x, sk);
          sk = fmaf(k4.y, s.y, sk);
          sk = fmaf(k4.z, s.z, sk);
          sk = fmaf(k4.w, s.w, sk);
        }
      }
#pragma unroll
      for (int w = 1; w < 8; w <<= 1) {
        sq += __shfl_xor_sync(0xffffffffu, sq, w);
        if (DELTA) sk += __shfl_xor_sync(0xffffffffu, sk, w);
      }
      const float u = fmaf(ev, v, -es * sk);
#pragma unroll
      for (int j = 0; j < CH / 4; ++j) {
        const int c = (j * 8 + g) * 4;
        const float4 k4 = *reinterpret_cast<const float4*>(&ks[c]);
        float4 s = S[k][j];
        s.x = fmaf(g_t, s.x, k4.x * u);
        s.y = fmaf(g_t, s.y, k4.y * u);
        s.z = fmaf(g_t, s.z, k4.z * u);
        s.w = fmaf(g_t, s.w, k4.w * u);
        if (ok && c < dim_p) __stcs(reinterpret_cast<float4*>(st + (long long)col * dim_p + c), s);
      }
      if (ok && g == 0) os[col] = fmaf(oq, sq, ou * u) + (p.skip ? p.skip[head] * v : 0.f);
    }
  }
  __syncthreads();
  if (!finish) {
    for (int c = threadIdx.x; c < p.vdim; c += kRecStepThreads) put(c, os[c]);
    return;
  }
  float ss = 0.f;
  for (int c = threadIdx.x; c < p.vdim; c += kRecStepThreads) ss += os[c] * os[c];
  ss = warp_sum(ss);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int w = 0; w < kRecStepThreads / 32; ++w) tot += red[w];
  const float inv = 1.f / sqrtf(tot / float(p.vdim) + p.eps);
  for (int c = threadIdx.x; c < p.vdim; c += kRecStepThreads) put(c, os[c] * inv * gs[c]);
}

template <int CH>
static int launch_rec_step(const NkbHeadRec& p, cudaStream_t s) {
  const dim3 grid(p.heads, p.batch), block(kRecStepThreads);
  const size_t smem = size_t(3 * p.vdim) * sizeof(float);
  using bf = __nv_bfloat16;
  if (p.b.ptr)
    return p.bf16 ? launch_pdl(head_rec_step_kernel<CH, true, bf>, grid, block, smem, s, p)
                  : launch_pdl(head_rec_step_kernel<CH, true, float>, grid, block, smem, s, p);
  return p.bf16 ? launch_pdl(head_rec_step_kernel<CH, false, bf>, grid, block, smem, s, p)
                : launch_pdl(head_rec_step_kernel<CH, false, float>, grid, block, smem, s, p);
}

// ------------------------------------------------------------------------------------------------ group norm
struct GroupNormParams {
  const void* y;            // [tokens, width]
  NkbProj g;                // [tokens, width]
  const float* w;
  void* out;
  long long units;          // parts of tokens
  int width, parts, warps, gate_act;      // warps: of a unit
  float eps;
};

// A unit (one part of one token) belongs to 1, 2, 4 or 8 warps; V elements per access: 8 of bf16, 4 of fp32 or split sums, or one.
// R > 0: a lane's R vectors stay in registers; R = 0: longer parts are read again for the result.
template <int V, int R, typename YT, typename OutT>
__global__ void __launch_bounds__(256) group_norm_kernel(const __grid_constant__ GroupNormParams p) {
  __shared__ float red[8];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, size = p.width / p.parts;
  const long long unit = blockIdx.x * (long long)(8 / p.warps) + warp / p.warps;
  const bool on = unit < p.units;
  const long long t = on ? unit / p.parts : 0;
  const int first = on ? int(unit % p.parts) * size : 0;
  const int i0 = (warp % p.warps * 32 + lane) * V, step = p.warps * 32 * V;
  griddep_wait();
  griddep_launch();
  const YT* y = reinterpret_cast<const YT*>(p.y) + t * p.width;
  OutT* out = reinterpret_cast<OutT*>(p.out) + t * p.width;
  const auto load = [&](float (&x)[V], int c) {
    float gt[V];
    if constexpr (V == 8) {
      ChanRaw<8> a, b;
      a.r = *reinterpret_cast<const uint4*>(y + c);
      b.load(p.g, t, c);
      a.get(x);
      b.get(gt);
    } else if constexpr (V == 4) {
      const float4 a = *reinterpret_cast<const float4*>(y + c), b = proj_load4(p.g, t, c);
      x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w;
      gt[0] = b.x; gt[1] = b.y; gt[2] = b.z; gt[3] = b.w;
    } else {
      x[0] = cast_in<YT>(y[c]);
      gt[0] = proj_load(p.g, t, c);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) {
      if (sizeof(OutT) == 2 && p.gate_act == ACT_SILU) x[e] *= silu_fast(gt[e]);
      else x[e] *= apply_act(gt[e], p.gate_act);
    }
  };
  const auto store = [&](const float (&x)[V], int c, float inv) {
    float r[V];
    if constexpr (V >= 4) {
#pragma unroll
      for (int e = 0; e < V; e += 4) {
        const float4 w = *reinterpret_cast<const float4*>(p.w + c + e);
        r[e] = x[e] * inv * w.x;
        r[e + 1] = x[e + 1] * inv * w.y;
        r[e + 2] = x[e + 2] * inv * w.z;
        r[e + 3] = x[e + 3] * inv * w.w;
      }
    } else {
      r[0] = x[0] * inv * p.w[c];
    }
    if constexpr (V == 8)
      *reinterpret_cast<uint4*>(out + c) =
          make_uint4(pack_bf16x2(r[0], r[1]), pack_bf16x2(r[2], r[3]), pack_bf16x2(r[4], r[5]), pack_bf16x2(r[6], r[7]));
    else if constexpr (V == 4 && sizeof(OutT) == 2)
      *reinterpret_cast<uint2*>(out + c) = make_uint2(pack_bf16x2(r[0], r[1]), pack_bf16x2(r[2], r[3]));
    else if constexpr (V == 4)
      *reinterpret_cast<float4*>(out + c) = make_float4(r[0], r[1], r[2], r[3]);
    else
      out[c] = cast_out<OutT>(r[0]);
  };
  float x[R > 0 ? R : 1][V], ss = 0.f;
  if constexpr (R > 0) {
#pragma unroll
    for (int k = 0; k < R; ++k) {
#pragma unroll
      for (int e = 0; e < V; ++e) x[k][e] = 0.f;
      if (on && i0 + k * step < size) load(x[k], first + i0 + k * step);
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(x[k][e], x[k][e], ss);
    }
  } else if (on) {
    for (int i = i0; i < size; i += step) {
      load(x[0], first + i);
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(x[0][e], x[0][e], ss);
    }
  }
  ss = warp_sum(ss);
  if (p.warps > 1) {
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    ss = 0.f;
    for (int w = 0; w < p.warps; ++w) ss += red[warp / p.warps * p.warps + w];
  }
  if (!on) return;
  const float inv = 1.f / sqrtf(ss / float(size) + p.eps);
  if constexpr (R > 0) {
#pragma unroll
    for (int k = 0; k < R; ++k)
      if (i0 + k * step < size) store(x[k], first + i0 + k * step, inv);
  } else {
    for (int i = i0; i < size; i += step) {
      load(x[0], first + i);
      store(x[0], first + i, inv);
    }
  }
}

template <int V, typename YT, typename OutT>
static int launch_group_norm(GroupNormParams p, cudaStream_t s) {
  const int size = p.width / p.parts, vectors = (size + V - 1) / V;
  // one warp per unit while that leaves four vectors or less per lane, more for long parts or few units
  p.warps = 1;
  while (p.warps < 8 && (vectors > 128 * p.warps || (p.units * p.warps < 148 * 16 && vectors > 32 * p.warps))) p.warps *= 2;
  const dim3 grid(unsigned((p.units + 8 / p.warps - 1) / (8 / p.warps))), block(256);
  const int rounds = (vectors + 32 * p.warps - 1) / (32 * p.warps);
  if (rounds <= 1) return launch_pdl(group_norm_kernel<V, 1, YT, OutT>, grid, block, 0, s, p);
  if (rounds <= 2) return launch_pdl(group_norm_kernel<V, 2, YT, OutT>, grid, block, 0, s, p);
  if (rounds <= 4) return launch_pdl(group_norm_kernel<V, 4, YT, OutT>, grid, block, 0, s, p);
  return launch_pdl(group_norm_kernel<V, 0, YT, OutT>, grid, block, 0, s, p);
}

static bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

static int head_rec_ok(const NkbHeadRec& p) {
  return p.heads >= 1 && p.heads <= 65535 && p.batch <= 65535 && p.groups >= 1 && p.heads % p.groups == 0 && p.dim >= 1 &&
         p.dim <= 256 && p.vdim >= 1 && p.vdim <= 1024 && p.x.ptr && p.a.ptr && p.rate && p.dt_bias && p.state &&
         p.context_lens && p.out;
}

}  // namespace nkb

using namespace nkb;

// x [tokens, channels] -> out; every row of the packed batch belongs to one of the sequences.
extern "C" int nkb_short_conv(const NkbProj* x, const float* w, const float* b, float* state, const int* slot_ids,
                              const int* q_start, const int* q_lens, const int* context_lens, void* out, int bf16, int batch,
                              int tokens, int channels, int taps, int act, void* stream) {
  if (batch <= 0 || tokens <= 0) return 0;
  if (channels < 1 || taps < 1 || taps > kMaxTaps || batch > 65535 || tokens > 4 * 65535 || act < 0 ||
      act >= ACT_CLAMPED || !q_start || !q_lens)
    return -2;
  ShortConvParams p{*x, w, b, state, slot_ids, q_start, q_lens, context_lens, out, batch, tokens, channels, taps, act, 0};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  int rc;
  if (bf16 && x->bf16 && channels % 4 == 0 && proj_vec4_ok(*x) && al16(out)) rc = launch_conv<4, __nv_bfloat16>(p, s);
  else rc = bf16 ? launch_conv<1, __nv_bfloat16>(p, s) : launch_conv<1, float>(p, s);
  if (rc) return rc;
  return launch_pdl(conv_state_kernel, dim3((channels + 255) / 256, batch), dim3(256), 0, s, p);
}

extern "C" int nkb_head_rec_scan(const NkbHeadRec* a, void* stream) {
  if (a->batch <= 0 || a->tokens <= 0) return 0;
  if (!head_rec_ok(*a) || a->x.splits != 1 || !a->q_start || !a->q_lens) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const bool async = a->bf16 && a->x.bf16 && ((a->dim | a->vdim | a->q_col | a->k_col | a->v_col) & 7) == 0 && al16(a->x.ptr) &&
                     a->x.ld % 8 == 0;
  if (a->dim <= 32) return launch_rec<4>(*a, async, s);
  if (a->dim <= 64) return launch_rec<8>(*a, async, s);
  if (a->dim <= 128) return launch_rec<16>(*a, async, s);
  return launch_rec<32>(*a, async, s);
}

extern "C" int nkb_head_rec_step(const NkbHeadRec* a, void* stream) {
  if (a->batch <= 0) return 0;
  if (!head_rec_ok(*a) || a->taps < 1 || a->taps > kMaxTaps || !a->conv_w || !a->conv_state || (a->norm_w && !a->g.ptr) ||
      a->gate_act < 0 || a->gate_act >= ACT_CLAMPED)
    return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dim <= 32) return launch_rec_step<4>(*a, s);
  if (a->dim <= 64) return launch_rec_step<8>(*a, s);
  if (a->dim <= 128) return launch_rec_step<16>(*a, s);
  return launch_rec_step<32>(*a, s);
}

extern "C" int nkb_gated_group_norm(const void* y, int y_bf16, const NkbProj* gate, int gate_act, const float* w, float eps,
                                    void* out, int out_bf16, int tokens, int width, int parts, void* stream) {
  if (tokens <= 0) return 0;
  if (width < 1 || parts < 1 || width % parts || gate_act < 0 || gate_act >= ACT_CLAMPED || !gate->ptr || !w) return -2;
  GroupNormParams p{y, *gate, w, out, (long long)tokens * parts, width, parts, 1, gate_act, eps};
  if (p.units > 0x7fffffffll) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  using bf = __nv_bfloat16;
  const int size = width / parts;
  if (y_bf16 && out_bf16 && gate->bf16 && size % 8 == 0 && al16(y) && al16(w) && al16(out) && al16(gate->ptr) && gate->ld % 8 == 0)
    return launch_group_norm<8, bf, bf>(p, s);
  if (!y_bf16 && size % 4 == 0 && al16(y) && al16(w) && al16(out) && proj_vec4_ok(*gate))
    return out_bf16 ? launch_group_norm<4, float, bf>(p, s) : launch_group_norm<4, float, float>(p, s);
  if (y_bf16) return out_bf16 ? launch_group_norm<1, bf, bf>(p, s) : -2;
  return out_bf16 ? launch_group_norm<1, float, bf>(p, s) : launch_group_norm<1, float, float>(p, s);
}
