// Linear attention with a decay per key channel (linear_attn.h) and the small operators around it:
//
//   token mix    m_i = h_t + (h_(t-1) - h_t) * mu_i for several mu_i; the last row of a sequence stays in its slot
//   low rank     z = W act(x) for a narrow x, in fp32
//   scan         any number of new tokens per sequence.  A CTA owns some columns of one head of one sequence for all of its
//                tokens; sixteen lanes share a set of columns, each holding every sixteenth group of four channels of
//                them in registers (three packed operations per two state elements and token).  A tile of tokens is copied
//                as it is while the previous one is multiplied, and turned into fp32 queries, keys, decays and values once
//                per CTA.  Sixteen partial sums (tokens x columns) are exchanged together by a transposing butterfly.
//   step         one new token per sequence (decode).  A CTA owns a head of a sequence, streams its state through registers
//                once, and computes everything around it itself: the low-rank decay, the norm of the head and its gate.
//   gate heads   out = scale * act(gate) * norm(head), for the scan's results and for attention heads (norm optional)
//
// The state of a sequence lives in its slot of a [slots, heads, vdim, dim_p] array (dim_p = dim rounded up to a multiple of
// 4); a sequence whose first new token has position 0 starts from zero, whatever the slot held.
#include "common.cuh"
#include "proj_src.cuh"
#include "activations.cuh"
#include "linear_attn.h"
#include "api.h"

namespace nkb {

// z already includes its bias.  sigmoid(z)^t = exp(-t * log(1 + exp(-z))), the logarithm in its stable form.  FAST uses the
// hardware's approximate exponential and logarithm (a few units in the last place of fp32), which bf16 inputs do not notice.
template <bool FAST>
__device__ __forceinline__ float decay_of(float z, int kind, float inv_tau) {
  if constexpr (FAST) {
    if (kind == NKB_DECAY_DOUBLE_EXP) return __expf(-__expf(z));
    return __expf(-inv_tau * (fmaxf(-z, 0.f) + __logf(1.f + __expf(-fabsf(z)))));
  }
  if (kind == NKB_DECAY_DOUBLE_EXP) return expf(-expf(z));
  return expf(-inv_tau * (fmaxf(-z, 0.f) + log1pf(expf(-fabsf(z)))));
}

template <int V>
__device__ __forceinline__ float4 load_channels(const NkbProj& s, long long row, int head_col, int c, int dim) {
  if constexpr (V == 4) return proj_load4(s, row, head_col + c);
  float4 r = make_float4(0.f, 0.f, 0.f, 0.f);
  if (c < dim) r.x = proj_load(s, row, head_col + c);
  if (c + 1 < dim) r.y = proj_load(s, row, head_col + c + 1);
  if (c + 2 < dim) r.z = proj_load(s, row, head_col + c + 2);
  if (c + 3 < dim) r.w = proj_load(s, row, head_col + c + 3);
  return r;
}

// ------------------------------------------------------------------------------------------------ token mix
struct TokenMixParams {
  const void* h;            // [tokens, width]
  const float* mu;          // [mixes, width]
  float* state;             // [slots, width]: the sequence's last row so far
  const int *slot_ids, *q_start, *q_lens, *context_lens;
  void* out;                // [mixes, tokens, width]
  int batch, tokens, width, mixes;
};
constexpr int kMixTokens = 8;     // tokens of a CTA in prompts
constexpr int kMaxMixes = 5;

// V consecutive elements in registers: 16 bytes of bf16 (V = 8), 16 bytes of fp32 (V = 4) or one element
template <int V, typename T>
__device__ __forceinline__ void load_run(float (&x)[V], const T* p) {
  if constexpr (V == 8) {
    const uint4 r = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 f = unpack_bf16x2(w[e]);
      x[2 * e] = f.x;
      x[2 * e + 1] = f.y;
    }
  } else if constexpr (V == 4) {
    const float4 r = *reinterpret_cast<const float4*>(p);
    x[0] = r.x; x[1] = r.y; x[2] = r.z; x[3] = r.w;
  } else {
    x[0] = cast_in<T>(*p);
  }
}
template <int V, typename T>
__device__ __forceinline__ void store_run(T* p, const float (&x)[V]) {
  if constexpr (V == 8) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(x[0], x[1]), pack_bf16x2(x[2], x[3]), pack_bf16x2(x[4], x[5]),
                                              pack_bf16x2(x[6], x[7]));
  } else if constexpr (V == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1], x[2], x[3]);
  } else {
    *p = cast_out<T>(x[0]);
  }
}

// A CTA owns a run of TB tokens and 128 V columns.  The first row of a portion reads what the last row writes, so the CTA
// that holds a sequence's last row also mixes its first one (before it stores), and the first row's own CTA leaves it out.
template <int V, int TB, typename T>
__global__ void __launch_bounds__(128) token_mix_kernel(const __grid_constant__ TokenMixParams p) {
  __shared__ int first_of[TB], last_of[TB];     // sequence that starts / ends at each token of the run, or -1
  const int t0 = blockIdx.y * TB, nt = min(TB, p.tokens - t0);
  const int c = (blockIdx.x * 128 + threadIdx.x) * V;
  if (threadIdx.x < TB) first_of[threadIdx.x] = last_of[threadIdx.x] = -1;
  griddep_wait();
  griddep_launch();
  __syncthreads();
  for (int b = threadIdx.x; b < p.batch; b += 128) {
    const int s = p.q_lens ? p.q_start[b] : b, n = p.q_lens ? p.q_lens[b] : 1;
    if (n <= 0) continue;
    if (s >= t0 && s < t0 + nt) first_of[s - t0] = b;
    if (s + n - 1 >= t0 && s + n - 1 < t0 + nt) last_of[s + n - 1 - t0] = b;
  }
  __syncthreads();
  if (c >= p.width) return;
  const T* h = reinterpret_cast<const T*>(p.h) + c;
  T* out = reinterpret_cast<T*>(p.out) + c;
  float mu[kMaxMixes][V];
#pragma unroll
  for (int m = 0; m < kMaxMixes; ++m)
    if (m < p.mixes)
#pragma unroll
      for (int j = 0; j < V; ++j) mu[m][j] = p.mu[(long long)m * p.width + c + j];
  auto emit = [&](long long t, const float (&prev)[V], const float (&x)[V]) {
#pragma unroll
    for (int m = 0; m < kMaxMixes; ++m)
      if (m < p.mixes) {
        float y[V];
#pragma unroll
        for (int j = 0; j < V; ++j) y[j] = fmaf(prev[j] - x[j], mu[m][j], x[j]);
        store_run<V, T>(out + ((long long)m * p.tokens + t) * p.width, y);
      }
  };
  float prev[V], x[V];
#pragma unroll
  for (int j = 0; j < V; ++j) prev[j] = 0.f;
  if (t0 > 0 && first_of[0] < 0) load_run<V, T>(prev, h + (t0 - 1ll) * p.width);
  load_run<V, T>(x, h + (long long)t0 * p.width);
#pragma unroll 1
  for (int i = 0; i < nt; ++i) {
    const long long t = t0 + i;
    float next[V];
#pragma unroll
    for (int j = 0; j < V; ++j) next[j] = 0.f;
    if (i + 1 < nt) load_run<V, T>(next, h + (t + 1) * p.width);
    const int bl = last_of[i];
    if (bl >= 0) {
      const int n = p.q_lens ? p.q_lens[bl] : 1, ctx = p.context_lens[bl];
      const long long start = p.q_lens ? p.q_start[bl] : bl;
      const bool active = ctx >= n;
      float* st = p.state + (long long)(p.slot_ids ? p.slot_ids[bl] : bl) * p.width + c;
      float head[V];
      if (n > 1) {
        emit(t, prev, x);
        load_run<V, T>(head, h + start * p.width);
      } else {
#pragma unroll
        for (int j = 0; j < V; ++j) head[j] = x[j];
      }
#pragma unroll
      for (int j = 0; j < V; ++j) prev[j] = active && ctx > n ? st[j] : 0.f;      // the row before the first one
      emit(start, prev, head);
      if (active)
#pragma unroll
        for (int j = 0; j < V; ++j) st[j] = x[j];
    } else if (first_of[i] < 0) {
      emit(t, prev, x);
    }
#pragma unroll
    for (int j = 0; j < V; ++j) {
      prev[j] = x[j];
      x[j] = next[j];
    }
  }
}

// ------------------------------------------------------------------------------------------------ low rank
// out[t, c] = sum_r w[c, r] * act(x[t, r]); 32 tokens x 64 outputs per CTA
template <typename WT>
__global__ void __launch_bounds__(256) low_rank_kernel(const __grid_constant__ NkbProj x, int act, const WT* __restrict__ w,
                                                       float* __restrict__ out, int tokens, int rank, int n) {
  constexpr int kR = 32;
  __shared__ float xs[32][kR + 1], ws[64][kR + 1];
  const int t0 = blockIdx.y * 32, c0 = blockIdx.x * 64;
  const int tr = threadIdx.x >> 5, tc = threadIdx.x & 31;
  float acc[4][2] = {};
  griddep_wait();
  griddep_launch();
  for (int r0 = 0; r0 < rank; r0 += kR) {
    for (int i = threadIdx.x; i < 32 * kR; i += 256) {
      const int t = t0 + i / kR, r = r0 + i % kR;
      xs[i / kR][i % kR] = t < tokens && r < rank ? apply_act(proj_load(x, t, r), act) : 0.f;
    }
    for (int i = threadIdx.x; i < 64 * kR; i += 256) {
      const int c = c0 + i / kR, r = r0 + i % kR;
      ws[i / kR][i % kR] = c < n && r < rank ? cast_in<WT>(w[(long long)c * rank + r]) : 0.f;
    }
    __syncthreads();
#pragma unroll 8
    for (int r = 0; r < kR; ++r) {
      const float w0 = ws[tc][r], w1 = ws[tc + 32][r];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float a = xs[tr + 8 * i][r];
        acc[i][0] = fmaf(a, w0, acc[i][0]);
        acc[i][1] = fmaf(a, w1, acc[i][1]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = t0 + tr + 8 * i;
    if (t >= tokens) continue;
#pragma unroll
    for (int j = 0; j < 2; ++j)
      if (c0 + tc + 32 * j < n) out[(long long)t * n + c0 + tc + 32 * j] = acc[i][j];
  }
}

// ------------------------------------------------------------------------------------------------ scan
constexpr int kScanThreads = 128;
constexpr int kScanLanes = 16;     // lanes that share the columns of a half warp

__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool on) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(on ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_all;" ::: "memory"); }

template <int CL, int NC>
struct ScanShape {
  static constexpr int TT = CL <= 8 ? 16 : 8;              // tokens per tile
  static constexpr int DP = kScanLanes * CL, COLS = 8 * NC;
  static constexpr int kWork = TT * (3 * DP + 2 * COLS) * 4;   // fp32 queries, keys, decays, values, outputs
  static constexpr int kRaw = TT * (DP * 8 + COLS * 2);        // decay logits fp32; queries, keys, values bf16
};

// CL: channels per lane (dim <= 16 CL), NC: columns per lane.  BONUS: read before the update.  ASYNC: queries, keys and
// values are bf16, the logits fp32, all in aligned runs of eight channels; otherwise tiles are read through NkbProj.
template <int CL, int NC, bool BONUS, bool ASYNC, typename OutT>
__global__ void __launch_bounds__(kScanThreads, CL <= 8 ? 4 : 1) linattn_scan_kernel(const __grid_constant__ NkbLinAttn p) {
  using S = ScanShape<CL, NC>;
  constexpr int TT = S::TT, DP = S::DP, COLS = S::COLS;
  constexpr int TB = kScanLanes / NC;               // tokens whose sums are exchanged together
  constexpr int QW = DP / 4;                        // threads that prepare one token's channels
  constexpr int BW = QW > 32 ? QW / 32 : 1;         // warps among them
  extern __shared__ __align__(16) uint8_t scan_s[];
  float(*qs)[DP] = reinterpret_cast<float(*)[DP]>(scan_s);
  float(*ks)[DP] = qs + TT;
  float(*as)[DP] = ks + TT;
  float(*vs)[COLS] = reinterpret_cast<float(*)[COLS]>(as + TT);
  float(*os)[COLS] = vs + TT;
  float(*zr)[DP] = reinterpret_cast<float(*)[DP]>(os + TT);
  __nv_bfloat16(*qr)[DP] = reinterpret_cast<__nv_bfloat16(*)[DP]>(zr + TT);
  __nv_bfloat16(*kr)[DP] = qr + TT;
  __nv_bfloat16(*vr)[COLS] = reinterpret_cast<__nv_bfloat16(*)[COLS]>(kr + TT);
  __shared__ float bon[TT][BW];
  __shared__ __align__(16) float zbs[DP], uus[BONUS ? DP : 4];
  const int head = blockIdx.y, b = blockIdx.z, col0 = blockIdx.x * COLS;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane & 15;
  const int cl0 = (warp * 2 + (lane >> 4)) * NC;    // first of this lane's columns within the CTA
  const int hq = head * p.dim, hv = head * p.vdim, dim_p = (p.dim + 3) / 4 * 4;
  // the channels this thread prepares are the same in every pass over a tile
  const int pc = (threadIdx.x % QW) * 4;
  for (int c = threadIdx.x; c < DP; c += kScanThreads) {
    zbs[c] = c < p.dim ? p.z_bias[hq + c] : 0.f;
    if (BONUS) uus[c] = c < p.dim ? p.bonus[hq + c] : 0.f;
  }
  griddep_wait();
  griddep_launch();
  const int n = p.q_lens[b], ctx = p.context_lens[b];
  if (n <= 0 || ctx < n) return;
  const long long row0 = p.q_start[b];
  const int slot = p.slot_ids ? p.slot_ids[b] : b;
  const bool fresh = ctx == n;
  float* st = p.state + (((long long)slot * p.heads + head) * p.vdim + col0 + cl0) * dim_p;

  auto fetch = [&](int t0) {
    if constexpr (ASYNC) {
#pragma unroll
      for (int i = 0; i < TT * DP / 8 / kScanThreads; ++i) {
        const int idx = threadIdx.x + i * kScanThreads, tok = idx / (DP / 8), c = idx % (DP / 8) * 8;
        const bool on = t0 + tok < n && c < p.dim;
        const long long r = on ? row0 + t0 + tok : row0;
        const int cc = on ? hq + c : hq;
        cp_async16(&qr[tok][c], reinterpret_cast<const __nv_bfloat16*>(p.q.ptr) + r * p.q.ld + cc, on);
        cp_async16(&kr[tok][c], reinterpret_cast<const __nv_bfloat16*>(p.k.ptr) + r * p.k.ld + cc, on);
        const float* z = reinterpret_cast<const float*>(p.z.ptr) + r * p.z.ld + cc;
        cp_async16(&zr[tok][c], z, on);
        cp_async16(&zr[tok][c + 4], z + (on ? 4 : 0), on);
      }
#pragma unroll
      for (int i = 0; i < (TT * COLS / 8 + kScanThreads - 1) / kScanThreads; ++i) {
        const int idx = threadIdx.x + i * kScanThreads, tok = idx / (COLS / 8), c = idx % (COLS / 8) * 8;
        if (idx < TT * COLS / 8) {
          const bool on = t0 + tok < n && col0 + c < p.vdim;
          const long long r = on ? row0 + t0 + tok : row0;
          cp_async16(&vr[tok][c], reinterpret_cast<const __nv_bfloat16*>(p.v.ptr) + r * p.v.ld + hv + (on ? col0 + c : 0), on);
        }
      }
      cp_async_commit();
    }
  };
  // the tile at t0 in fp32; tokens past the end keep the state (decay one, key zero)
  auto prepare = [&](int t0) {
#pragma unroll
    for (int i = 0; i < TT * QW / kScanThreads; ++i) {
      const int tok = (threadIdx.x + i * kScanThreads) / QW;
      const bool on = t0 + tok < n && pc < p.dim;
      float q[4] = {0.f, 0.f, 0.f, 0.f}, k[4] = {0.f, 0.f, 0.f, 0.f}, a[4] = {1.f, 1.f, 1.f, 1.f};
      if (on) {
        float4 q4, k4, z4;
        if constexpr (ASYNC) {
          const uint2 qu = *reinterpret_cast<const uint2*>(&qr[tok][pc]), ku = *reinterpret_cast<const uint2*>(&kr[tok][pc]);
          const float2 q0 = unpack_bf16x2(qu.x), q1 = unpack_bf16x2(qu.y), k0 = unpack_bf16x2(ku.x), k1 = unpack_bf16x2(ku.y);
          q4 = make_float4(q0.x, q0.y, q1.x, q1.y);
          k4 = make_float4(k0.x, k0.y, k1.x, k1.y);
          z4 = *reinterpret_cast<const float4*>(&zr[tok][pc]);
        } else {
          q4 = load_channels<1>(p.q, row0 + t0 + tok, hq, pc, p.dim);
          k4 = load_channels<1>(p.k, row0 + t0 + tok, hq, pc, p.dim);
          z4 = load_channels<1>(p.z, row0 + t0 + tok, hq, pc, p.dim);
        }
        const float qv[4] = {q4.x, q4.y, q4.z, q4.w}, kv[4] = {k4.x, k4.y, k4.z, k4.w}, zv[4] = {z4.x, z4.y, z4.z, z4.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          q[e] = qv[e] * p.q_scale;
          k[e] = kv[e];
          a[e] = decay_of<ASYNC>(zv[e] + zbs[pc + e], p.decay, p.inv_tau);
        }
      }
      *reinterpret_cast<float4*>(&qs[tok][pc]) = make_float4(q[0], q[1], q[2], q[3]);
      *reinterpret_cast<float4*>(&ks[tok][pc]) = make_float4(k[0], k[1], k[2], k[3]);
      *reinterpret_cast<float4*>(&as[tok][pc]) = make_float4(a[0], a[1], a[2], a[3]);
      if constexpr (BONUS) {
        const float4 u4 = *reinterpret_cast<const float4*>(&uus[pc]);
        float s = q[0] * u4.x * k[0] + q[1] * u4.y * k[1] + q[2] * u4.z * k[2] + q[3] * u4.w * k[3];
#pragma unroll
        for (int w = (QW < 32 ? QW : 32) / 2; w > 0; w >>= 1) s += __shfl_xor_sync(0xffffffffu, s, w);
        if (threadIdx.x % (QW < 32 ? QW : 32) == 0) bon[tok][BW > 1 ? (threadIdx.x % QW) / 32 : 0] = s;
      }
    }
#pragma unroll
    for (int i = 0; i < (TT * COLS + kScanThreads - 1) / kScanThreads; ++i) {
      const int idx = threadIdx.x + i * kScanThreads, tok = idx / COLS, c = idx % COLS;
      if constexpr (ASYNC) {
        vs[tok][c] = __bfloat162float(vr[tok][c]);
      } else {
        vs[tok][c] = t0 + tok < n && col0 + c < p.vdim ? proj_load(p.v, row0 + t0 + tok, hv + col0 + c) : 0.f;
      }
    }
  };
  fetch(0);

  // channels of this lane: groups of four, group j at (j * 16 + g) * 4
  float2 D[NC][CL / 2];
#pragma unroll
  for (int k = 0; k < NC; ++k) {
    const bool ok = col0 + cl0 + k < p.vdim;
#pragma unroll
    for (int j = 0; j < CL / 4; ++j) {
      const int c = (j * kScanLanes + g) * 4;
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!fresh && ok && c < dim_p) x = *reinterpret_cast<const float4*>(st + (long long)k * dim_p + c);
      D[k][2 * j] = make_float2(x.x, x.y);
      D[k][2 * j + 1] = make_float2(x.z, x.w);
    }
  }

#pragma unroll 1
  for (int t0 = 0; t0 < n; t0 += TT) {
    cp_async_wait_all();
    __syncthreads();                                 // the raw tile is there; nobody reads the fp32 tile or os any more
    prepare(t0);
    __syncthreads();
    if (t0 + TT < n) fetch(t0 + TT);
#pragma unroll 1
    for (int h = 0; h < TT; h += TB) {
      if (t0 + h >= n) break;
      float po[kScanLanes];                          // [token][column]
#pragma unroll
      for (int tt = 0; tt < TB; ++tt) {
        float v[NC];
        if constexpr (NC >= 4) {
#pragma unroll
          for (int k = 0; k < NC; k += 4) {
            const float4 x = *reinterpret_cast<const float4*>(&vs[h + tt][cl0 + k]);
            v[k] = x.x; v[k + 1] = x.y; v[k + 2] = x.z; v[k + 3] = x.w;
          }
        } else {
#pragma unroll
          for (int k = 0; k < NC; ++k) v[k] = vs[h + tt][cl0 + k];
        }
        float2 o[NC];
#pragma unroll
        for (int k = 0; k < NC; ++k) o[k] = make_float2(0.f, 0.f);
#pragma unroll
        for (int j = 0; j < CL / 4; ++j) {
          const int c = (j * kScanLanes + g) * 4;
          const float4 q4 = *reinterpret_cast<const float4*>(&qs[h + tt][c]);
          const float4 k4 = *reinterpret_cast<const float4*>(&ks[h + tt][c]);
          const float4 a4 = *reinterpret_cast<const float4*>(&as[h + tt][c]);
          const float2 q2[2] = {make_float2(q4.x, q4.y), make_float2(q4.z, q4.w)};
          const float2 k2[2] = {make_float2(k4.x, k4.y), make_float2(k4.z, k4.w)};
          const float2 a2[2] = {make_float2(a4.x, a4.y), make_float2(a4.z, a4.w)};
#pragma unroll
          for (int k = 0; k < NC; ++k) {
            const float2 v2 = make_float2(v[k], v[k]);
#pragma unroll
            for (int i = 0; i < 2; ++i) {
              float2& d = D[k][2 * j + i];
              if constexpr (BONUS) o[k] = ffma2(q2[i], d, o[k]);
              d = ffma2(a2[i], d, fmul2(k2[i], v2));
              if constexpr (!BONUS) o[k] = ffma2(q2[i], d, o[k]);
            }
          }
        }
#pragma unroll
        for (int k = 0; k < NC; ++k) po[tt * NC + k] = o[k].x + o[k].y;
      }
      // sixteen lanes x sixteen sums: lane g ends with sum g, i.e. token g / NC, column g % NC
#pragma unroll
      for (int w = kScanLanes / 2; w > 0; w >>= 1) {
#pragma unroll
        for (int i = 0; i < w; ++i) {
          const float keep = (g & w) ? po[w + i] : po[i], send = (g & w) ? po[i] : po[w + i];
          po[i] = keep + __shfl_xor_sync(0xffffffffu, send, w);
        }
      }
      os[h + g / NC][cl0 + g % NC] = po[0];
    }
    __syncthreads();
    OutT* out = reinterpret_cast<OutT*>(p.heads_out);
#pragma unroll
    for (int i = 0; i < (TT * COLS + kScanThreads - 1) / kScanThreads; ++i) {
      const int idx = threadIdx.x + i * kScanThreads, tok = idx / COLS, c = idx % COLS;
      if (t0 + tok < n && col0 + c < p.vdim) {
        float r = os[tok][c];
        if constexpr (BONUS) {
          float bb = bon[tok][0];
#pragma unroll
          for (int w = 1; w < BW; ++w) bb += bon[tok][w];
          r = fmaf(bb, vs[tok][c], r);
        }
        out[(row0 + t0 + tok) * p.heads * p.vdim + hv + col0 + c] = cast_out<OutT>(r);
      }
    }
  }
#pragma unroll
  for (int k = 0; k < NC; ++k)
#pragma unroll
    for (int j = 0; j < CL / 4; ++j) {
      const int c = (j * kScanLanes + g) * 4;
      if (col0 + cl0 + k < p.vdim && c < dim_p)
        *reinterpret_cast<float4*>(st + (long long)k * dim_p + c) =
            make_float4(D[k][2 * j].x, D[k][2 * j].y, D[k][2 * j + 1].x, D[k][2 * j + 1].y);
    }
}

// ------------------------------------------------------------------------------------------------ gate heads
struct GateHeadsParams {
  const void* x;            // token t, head h: x + t * ld_token + h * ld_head
  long long ld_token, ld_head;
  NkbProj g;                // [tokens, heads * width], or [tokens, heads]: one gate per head
  const float* norm_w;      // nullptr: the head is not normed; otherwise element h * norm_stride + j
  void* out;
  long long out_ld, rows;   // rows = tokens * heads
  int gate_act, norm_stride, heads, width, head_gate;
  float eps, scale;
};

template <typename T>
__device__ __forceinline__ float4 load4_as(const T* p) {
  if constexpr (sizeof(T) == 2) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
    return make_float4(a.x, a.y, b.x, b.y);
  } else {
    return *reinterpret_cast<const float4*>(p);
  }
}

// One warp per (token, head).  VEC: width a multiple of 4, at most 128, everything aligned: a lane holds its four elements.
template <bool VEC, typename XT, typename OutT>
__global__ void __launch_bounds__(256) gate_heads_kernel(const __grid_constant__ GateHeadsParams p) {
  griddep_wait();
  griddep_launch();
  const long long i = (blockIdx.x * 256ll + threadIdx.x) >> 5;
  const int lane = threadIdx.x & 31;
  if (i >= p.rows) return;
  const long long t = i / p.heads;
  const int h = int(i % p.heads);
  const XT* x = reinterpret_cast<const XT*>(p.x) + t * p.ld_token + h * p.ld_head;
  OutT* out = reinterpret_cast<OutT*>(p.out) + t * p.out_ld + (long long)h * p.width;
  const float* w = p.norm_w ? p.norm_w + (long long)h * p.norm_stride : nullptr;
  if constexpr (VEC) {
    const int c = lane * 4;
    const bool on = c < p.width;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f), gt = v, ww = make_float4(1.f, 1.f, 1.f, 1.f);
    if (on) {
      v = load4_as<XT>(x + c);
      if (p.head_gate) gt.x = gt.y = gt.z = gt.w = proj_load(p.g, t, h);
      else gt = proj_load4(p.g, t, h * p.width + c);
      if (w) ww = *reinterpret_cast<const float4*>(w + c);
    }
    float inv = p.scale;
    if (w) inv *= 1.f / sqrtf(warp_sum(v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w) / float(p.width) + p.eps);
    if (on) {
      v.x *= inv * ww.x * apply_act(gt.x, p.gate_act);
      v.y *= inv * ww.y * apply_act(gt.y, p.gate_act);
      v.z *= inv * ww.z * apply_act(gt.z, p.gate_act);
      v.w *= inv * ww.w * apply_act(gt.w, p.gate_act);
      if constexpr (sizeof(OutT) == 2)
        *reinterpret_cast<uint2*>(out + c) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
      else
        *reinterpret_cast<float4*>(out + c) = v;
    }
    return;
  }
  float inv = p.scale;
  if (w) {
    float ss = 0.f;
    for (int c = lane; c < p.width; c += 32) {
      const float v = cast_in<XT>(x[c]);
      ss += v * v;
    }
    inv *= 1.f / sqrtf(warp_sum(ss) / float(p.width) + p.eps);
  }
  for (int c = lane; c < p.width; c += 32)
    out[c] = cast_out<OutT>(cast_in<XT>(x[c]) * inv * (w ? w[c] : 1.f) *
                            apply_act(proj_load(p.g, t, p.head_gate ? h : h * p.width + c), p.gate_act));
}

// bf16 heads of a multiple of eight elements, at most 256: L lanes share a head, a lane holds eight consecutive elements of
// two heads and loads all of them first.
template <int L, int GATE, bool NORM, bool HEAD = false>
__global__ void __launch_bounds__(256) gate_heads8_kernel(const __grid_constant__ GateHeadsParams p) {
  using bf = __nv_bfloat16;
  const int per = 256 / L, lane = threadIdx.x & (L - 1), c = lane * 8;
  const bool on = c < p.width;
  griddep_wait();
  griddep_launch();
  uint4 xr[2], gr[2], gr2[2];
  float hg[2];
  int tok[2], hd[2];
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    const long long i = (blockIdx.x * 2ll + u) * per + threadIdx.x / L;
    const bool live = i < p.rows && on;
    tok[u] = live ? int(i) / p.heads : -1;
    hd[u] = live ? int(i) % p.heads : 0;
    xr[u] = gr[u] = gr2[u] = make_uint4(0u, 0u, 0u, 0u);
    hg[u] = 0.f;
    if (live) {
      const int col = hd[u] * p.width + c;
      xr[u] = *reinterpret_cast<const uint4*>(reinterpret_cast<const bf*>(p.x) + tok[u] * p.ld_token + hd[u] * p.ld_head + c);
      if constexpr (HEAD) {
        hg[u] = proj_load(p.g, tok[u], hd[u]);
      } else if (p.g.bf16) {
        gr[u] = *reinterpret_cast<const uint4*>(reinterpret_cast<const bf*>(p.g.ptr) + tok[u] * p.g.ld + col);
      } else {
        const float4 lo = proj_load4(p.g, tok[u], col), hi = proj_load4(p.g, tok[u], col + 4);
        gr[u] = make_uint4(__float_as_uint(lo.x), __float_as_uint(lo.y), __float_as_uint(lo.z), __float_as_uint(lo.w));
        gr2[u] = make_uint4(__float_as_uint(hi.x), __float_as_uint(hi.y), __float_as_uint(hi.z), __float_as_uint(hi.w));
      }
    }
  }
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    float x[8], g[8];
    const uint32_t rw[4] = {xr[u].x, xr[u].y, xr[u].z, xr[u].w};
    const uint32_t gw[8] = {gr[u].x, gr[u].y, gr[u].z, gr[u].w, gr2[u].x, gr2[u].y, gr2[u].z, gr2[u].w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 f = unpack_bf16x2(rw[e]);
      x[2 * e] = f.x;
      x[2 * e + 1] = f.y;
    }
    if constexpr (HEAD) {
#pragma unroll
      for (int e = 0; e < 8; ++e) g[e] = hg[u];
    } else if (p.g.bf16) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 f = unpack_bf16x2(gw[e]);
        g[2 * e] = f.x;
        g[2 * e + 1] = f.y;
      }
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) g[e] = __uint_as_float(gw[e]);
    }
    float inv = p.scale;
    if constexpr (NORM) {
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < 8; ++e) ss += x[e] * x[e];
#pragma unroll
      for (int w = L / 2; w > 0; w >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, w);
      inv *= 1.f / sqrtf(ss / float(p.width) + p.eps);
    }
    if (tok[u] >= 0) {
      if constexpr (NORM) {
        const float* w = p.norm_w + (long long)hd[u] * p.norm_stride + c;
        const float4 lo = *reinterpret_cast<const float4*>(w), hi = *reinterpret_cast<const float4*>(w + 4);
        const float ww[8] = {lo.x, lo.y, lo.z, lo.w, hi.x, hi.y, hi.z, hi.w};
#pragma unroll
        for (int e = 0; e < 8; ++e) x[e] *= ww[e];
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        if constexpr (GATE == ACT_SILU) x[e] *= inv * g[e] * __fdividef(1.f, 1.f + __expf(-g[e]));
        else if constexpr (GATE == ACT_SIGMOID) x[e] *= inv * __fdividef(1.f, 1.f + __expf(-g[e]));
        else x[e] *= inv * apply_act(g[e], p.gate_act);
      }
      *reinterpret_cast<uint4*>(reinterpret_cast<bf*>(p.out) + tok[u] * p.out_ld + (long long)hd[u] * p.width + c) =
          make_uint4(pack_bf16x2(x[0], x[1]), pack_bf16x2(x[2], x[3]), pack_bf16x2(x[4], x[5]), pack_bf16x2(x[6], x[7]));
    }
  }
}

static bool al(const void* p, int bytes) { return (reinterpret_cast<uintptr_t>(p) & (bytes - 1)) == 0; }

template <int L>
static int launch_gate_heads8(const GateHeadsParams& p, cudaStream_t s) {
  const dim3 grid(unsigned((p.rows + 512 / L - 1) / (512 / L))), block(256);
  if (p.head_gate) {
    if (p.norm_w) return launch_pdl(gate_heads8_kernel<L, ACT_NONE, true, true>, grid, block, 0, s, p);
    if (p.gate_act == ACT_SIGMOID) return launch_pdl(gate_heads8_kernel<L, ACT_SIGMOID, false, true>, grid, block, 0, s, p);
    return launch_pdl(gate_heads8_kernel<L, ACT_NONE, false, true>, grid, block, 0, s, p);
  }
  if (p.norm_w) {
    if (p.gate_act == ACT_SILU) return launch_pdl(gate_heads8_kernel<L, ACT_SILU, true>, grid, block, 0, s, p);
    return launch_pdl(gate_heads8_kernel<L, ACT_NONE, true>, grid, block, 0, s, p);
  }
  if (p.gate_act == ACT_SIGMOID) return launch_pdl(gate_heads8_kernel<L, ACT_SIGMOID, false>, grid, block, 0, s, p);
  return launch_pdl(gate_heads8_kernel<L, ACT_NONE, false>, grid, block, 0, s, p);
}

static int launch_gate_heads(const GateHeadsParams& p, int x_bf16, int out_bf16, cudaStream_t s) {
  const int xb = x_bf16 ? 8 : 16, ob = out_bf16 ? 8 : 16;
  const bool vec = p.width % 4 == 0 && p.width <= 128 && p.ld_token % 4 == 0 && p.ld_head % 4 == 0 && p.out_ld % 4 == 0 &&
                   al(p.x, xb) && al(p.out, ob) && (p.head_gate || proj_vec4_ok(p.g)) &&
                   (!p.norm_w || (al(p.norm_w, 16) && p.norm_stride % 4 == 0));
  const dim3 grid(unsigned((p.rows + 7) / 8)), block(256);
  using bf = __nv_bfloat16;
  if (x_bf16 && out_bf16 && p.width % 8 == 0 && p.width <= 256 && p.rows < (1ll << 30) && p.ld_token % 8 == 0 &&
      p.ld_head % 8 == 0 && p.out_ld % 8 == 0 && al(p.x, 16) && al(p.out, 16) && (p.head_gate || proj_vec4_ok(p.g)) &&
      (p.head_gate || !p.g.bf16 || (al(p.g.ptr, 16) && p.g.ld % 8 == 0))) {
    if (!p.norm_w || (al(p.norm_w, 16) && p.norm_stride % 4 == 0)) {
      if (p.width <= 64) return launch_gate_heads8<8>(p, s);
      if (p.width <= 128) return launch_gate_heads8<16>(p, s);
      return launch_gate_heads8<32>(p, s);
    }
  }
  if (x_bf16 && out_bf16)
    return vec ? launch_pdl(gate_heads_kernel<true, bf, bf>, grid, block, 0, s, p)
               : launch_pdl(gate_heads_kernel<false, bf, bf>, grid, block, 0, s, p);
  if (!x_bf16 && !out_bf16)
    return vec ? launch_pdl(gate_heads_kernel<true, float, float>, grid, block, 0, s, p)
               : launch_pdl(gate_heads_kernel<false, float, float>, grid, block, 0, s, p);
  return -2;
}

// ------------------------------------------------------------------------------------------------ step
constexpr int kStepThreads = 256;
constexpr int kStepBlocks = 4;      // column blocks of 32 in flight

template <int CH, bool BONUS, typename OutT>
__global__ void __launch_bounds__(kStepThreads) linattn_step_kernel(const __grid_constant__ NkbLinAttn p) {
  constexpr int D8 = 8 * CH;
  __shared__ __align__(16) float qs[D8], ks[D8], as[D8], us[BONUS ? D8 : 4];
  __shared__ float red[kStepThreads / 32];
  extern __shared__ float dyn[];                    // v, o, norm weight times gate [vdim] each, low-rank input [rank]
  float* vs = dyn;
  float* os = dyn + p.vdim;
  float* gs = os + p.vdim;
  float* xs = gs + p.vdim;
  const int head = blockIdx.x, b = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane & 7;
  const int cl = warp * 4 + (lane >> 3);
  const int hq = head * p.dim, hv = head * p.vdim, dim_p = (p.dim + 3) / 4 * 4;
  griddep_wait();
  griddep_launch();
  OutT* out = reinterpret_cast<OutT*>(p.out) + b * p.out_ld + hv;
  const int ctx = p.context_lens[b];
  if (ctx <= 0) {
    for (int c = threadIdx.x; c < p.vdim; c += kStepThreads) out[c] = cast_out<OutT>(0.f);
    return;
  }
  const int slot = p.slot_ids ? p.slot_ids[b] : b;
  const bool fresh = ctx == 1;
  float* st = p.state + ((long long)slot * p.heads + head) * p.vdim * dim_p;
  const int nblk = (p.vdim + 31) / 32;
  for (int b0 = 0; b0 < nblk; b0 += kStepBlocks) {
    float4 S[kStepBlocks][CH / 4];
#pragma unroll
    for (int k = 0; k < kStepBlocks; ++k) {
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
      for (int r = threadIdx.x; r < p.rank; r += kStepThreads) xs[r] = apply_act(proj_load(p.z, b, r), p.z_act);
      for (int c = threadIdx.x; c < p.vdim; c += kStepThreads) {
        vs[c] = proj_load(p.v, b, hv + c);
        gs[c] = p.norm_w[(long long)head * p.norm_stride + c] * apply_act(proj_load(p.g, b, hv + c), p.gate_act);
      }
      for (int c = threadIdx.x; c < D8; c += kStepThreads) {
        const bool on = c < p.dim;
        const float q = on ? proj_load(p.q, b, hq + c) * p.q_scale : 0.f, k = on ? proj_load(p.k, b, hq + c) : 0.f;
        qs[c] = q;
        ks[c] = k;
        if (BONUS) us[c] = on ? p.bonus[hq + c] * k : 0.f;
      }
      __syncthreads();
      // the decay logit of a channel by P neighbouring lanes
      constexpr int P = kStepThreads / D8 > 0 ? kStepThreads / D8 : 1;
      const int c = threadIdx.x / P, part = threadIdx.x % P;
      float z = 0.f;
      if (c < p.dim) {
        if (!p.w2) {
          z = part == 0 ? proj_load(p.z, b, hq + c) : 0.f;
        } else if (p.w2_bf16) {
          const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(p.w2) + (long long)(hq + c) * p.rank;
          if ((p.rank & 7) == 0 && (reinterpret_cast<uintptr_t>(p.w2) & 15) == 0) {
            for (int r = part * 8; r < p.rank; r += P * 8) {
              const uint4 u = *reinterpret_cast<const uint4*>(w + r);
              const uint32_t uw[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                const float2 f = unpack_bf16x2(uw[e]);
                z = fmaf(f.x, xs[r + 2 * e], z);
                z = fmaf(f.y, xs[r + 2 * e + 1], z);
              }
            }
          } else {
            for (int r = part; r < p.rank; r += P) z = fmaf(__bfloat162float(w[r]), xs[r], z);
          }
        } else {
          const float* w = reinterpret_cast<const float*>(p.w2) + (long long)(hq + c) * p.rank;
          for (int r = part; r < p.rank; r += P) z = fmaf(w[r], xs[r], z);
        }
      }
#pragma unroll
      for (int w = P / 2; w > 0; w >>= 1) z += __shfl_xor_sync(0xffffffffu, z, w);
      if (part == 0 && c < D8) as[c] = c < p.dim ? decay_of<sizeof(OutT) == 2>(z + p.z_bias[hq + c], p.decay, p.inv_tau) : 1.f;
      __syncthreads();
    }
#pragma unroll
    for (int k = 0; k < kStepBlocks; ++k) {
      const int col = (b0 + k) * 32 + cl;
      const bool ok = col < p.vdim;
      const float v = ok ? vs[col] : 0.f;
      float o = 0.f;
#pragma unroll
      for (int j = 0; j < CH / 4; ++j) {
        const int c = (j * 8 + g) * 4;
        const float4 a4 = *reinterpret_cast<const float4*>(&as[c]), k4 = *reinterpret_cast<const float4*>(&ks[c]);
        const float4 q4 = *reinterpret_cast<const float4*>(&qs[c]);
        float4 s = S[k][j];
        if constexpr (BONUS) {
          const float4 u4 = *reinterpret_cast<const float4*>(&us[c]);
          o = fmaf(q4.x, fmaf(u4.x, v, s.x), o);
          o = fmaf(q4.y, fmaf(u4.y, v, s.y), o);
          o = fmaf(q4.z, fmaf(u4.z, v, s.z), o);
          o = fmaf(q4.w, fmaf(u4.w, v, s.w), o);
        }
        s.x = fmaf(a4.x, s.x, k4.x * v);
        s.y = fmaf(a4.y, s.y, k4.y * v);
        s.z = fmaf(a4.z, s.z, k4.z * v);
        s.w = fmaf(a4.w, s.w, k4.w * v);
        if constexpr (!BONUS) {
          o = fmaf(q4.x, s.x, o);
          o = fmaf(q4.y, s.y, o);
          o = fmaf(q4.z, s.z, o);
          o = fmaf(q4.w, s.w, o);
        }
        if (ok && c < dim_p) __stcs(reinterpret_cast<float4*>(st + (long long)col * dim_p + c), s);
      }
      o += __shfl_xor_sync(0xffffffffu, o, 1);
      o += __shfl_xor_sync(0xffffffffu, o, 2);
      o += __shfl_xor_sync(0xffffffffu, o, 4);
      if (ok && g == 0) os[col] = o;
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = threadIdx.x; c < p.vdim; c += kStepThreads) ss += os[c] * os[c];
  ss = warp_sum(ss);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int w = 0; w < kStepThreads / 32; ++w) tot += red[w];
  const float inv = p.out_scale / sqrtf(tot / float(p.vdim) + p.eps);
  for (int c = threadIdx.x; c < p.vdim; c += kStepThreads) out[c] = cast_out<OutT>(os[c] * inv * gs[c]);
}

template <int CL, int NC, bool BONUS, bool ASYNC, typename OutT>
static int launch_scan_one(const NkbLinAttn& p, cudaStream_t s) {
  using S = ScanShape<CL, NC>;
  constexpr int smem = S::kWork + (ASYNC ? S::kRaw : 0);
  auto kernel = linattn_scan_kernel<CL, NC, BONUS, ASYNC, OutT>;
  static bool attr_set[64] = {false};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -1;
  if (!attr_set[dev]) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return int(e);
    attr_set[dev] = true;
  }
  return launch_pdl(kernel, dim3((p.vdim + 8 * NC - 1) / (8 * NC), p.heads, p.batch), dim3(kScanThreads), size_t(smem), s, p);
}
template <int CL, int NC>
static int launch_scan_form(const NkbLinAttn& p, bool async, cudaStream_t s) {
  using bf = __nv_bfloat16;
  if (async)
    return p.bonus ? launch_scan_one<CL, NC, true, true, bf>(p, s) : launch_scan_one<CL, NC, false, true, bf>(p, s);
  if (p.bf16)
    return p.bonus ? launch_scan_one<CL, NC, true, false, bf>(p, s) : launch_scan_one<CL, NC, false, false, bf>(p, s);
  return p.bonus ? launch_scan_one<CL, NC, true, false, float>(p, s) : launch_scan_one<CL, NC, false, false, float>(p, s);
}
// More columns per lane mean fewer shared-memory reads per state element, fewer mean more warps to hide latency with.
template <int CL>
static int launch_scan(const NkbLinAttn& p, bool async, cudaStream_t s) {
  const auto ctas = [&](int cols) { return (long long)p.batch * p.heads * ((p.vdim + cols - 1) / cols); };
  if constexpr (CL <= 8)
    if (ctas(64) >= 2 * 148) return launch_scan_form<CL, 8>(p, async, s);
  if (ctas(32) >= 200) return launch_scan_form<CL, 4>(p, async, s);
  return launch_scan_form<CL, 2>(p, async, s);
}
template <int CH, bool BONUS>
static int launch_step_form(const NkbLinAttn& p, cudaStream_t s) {
  const dim3 grid(p.heads, p.batch);
  const size_t smem = size_t(3 * p.vdim + p.rank) * sizeof(float);
  return p.bf16 ? launch_pdl(linattn_step_kernel<CH, BONUS, __nv_bfloat16>, grid, dim3(kStepThreads), smem, s, p)
                : launch_pdl(linattn_step_kernel<CH, BONUS, float>, grid, dim3(kStepThreads), smem, s, p);
}
template <int CH>
static int launch_step(const NkbLinAttn& p, cudaStream_t s) {
  return p.bonus ? launch_step_form<CH, true>(p, s) : launch_step_form<CH, false>(p, s);
}

static int linattn_ok(const NkbLinAttn& p) {
  return p.heads >= 1 && p.heads <= 65535 && p.batch <= 65535 && p.dim >= 1 && p.dim <= 256 && p.vdim >= 1 &&
         p.vdim <= 1024 && p.rank >= 0 && p.rank <= 4096 && (p.rank == 0) == (p.w2 == nullptr) && p.state && p.context_lens &&
         p.norm_w && p.z_bias && p.out && p.g.ptr && (p.decay == NKB_DECAY_SIGMOID || p.decay == NKB_DECAY_DOUBLE_EXP) &&
         p.gate_act >= 0 && p.gate_act < ACT_COUNT && p.z_act >= 0 && p.z_act < ACT_COUNT;
}

}  // namespace nkb

using namespace nkb;

// Every row of the packed batch belongs to one of the sequences.  The decay logits are finished (w2 == nullptr).
extern "C" int nkb_linattn_scan(const NkbLinAttn* a, void* stream) {
  if (a->batch <= 0 || a->tokens <= 0) return 0;
  if (!linattn_ok(*a) || a->w2 || !a->heads_out || !a->q_start || !a->q_lens) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const auto bf_ok = [](const NkbProj& x) { return x.bf16 && al(x.ptr, 16) && x.ld % 8 == 0; };
  const bool async = a->bf16 && a->dim % 8 == 0 && a->vdim % 8 == 0 && bf_ok(a->q) && bf_ok(a->k) && bf_ok(a->v) &&
                     !a->z.bf16 && a->z.splits == 1 && al(a->z.ptr, 16) && a->z.ld % 4 == 0;
  int rc = a->dim <= 64 ? launch_scan<4>(*a, async, s)
                        : (a->dim <= 128 ? launch_scan<8>(*a, async, s) : launch_scan<16>(*a, async, s));
  if (rc) return rc;
  GateHeadsParams p{};
  p.x = a->heads_out;
  p.ld_token = (long long)a->heads * a->vdim;
  p.ld_head = a->vdim;
  p.g = a->g; p.norm_w = a->norm_w; p.out = a->out; p.out_ld = a->out_ld;
  p.rows = (long long)a->tokens * a->heads;
  p.gate_act = a->gate_act; p.norm_stride = a->norm_stride; p.heads = a->heads; p.width = a->vdim;
  p.eps = a->eps; p.scale = a->out_scale;
  return launch_gate_heads(p, a->bf16, a->bf16, s);
}

extern "C" int nkb_linattn_step(const NkbLinAttn* a, void* stream) {
  if (a->batch <= 0) return 0;
  if (!linattn_ok(*a)) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dim <= 32) return launch_step<4>(*a, s);
  if (a->dim <= 64) return launch_step<8>(*a, s);
  if (a->dim <= 128) return launch_step<16>(*a, s);
  return launch_step<32>(*a, s);
}

extern "C" int nkb_low_rank(const NkbProj* x, int act, const void* w, int w_bf16, float* out, int tokens, int rank, int n,
                            void* stream) {
  if (tokens <= 0 || n <= 0) return 0;
  if (rank < 1 || act < 0 || act >= ACT_COUNT || (tokens + 31) / 32 > 65535) return -2;
  const dim3 grid((n + 63) / 64, (tokens + 31) / 32);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return w_bf16 ? launch_pdl(low_rank_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, *x, act,
                             reinterpret_cast<const __nv_bfloat16*>(w), out, tokens, rank, n)
                : launch_pdl(low_rank_kernel<float>, grid, dim3(256), 0, s, *x, act, reinterpret_cast<const float*>(w), out,
                             tokens, rank, n);
}

// q_lens == nullptr: one new token per sequence, row b of h belongs to sequence b.
extern "C" int nkb_token_mix(const void* h, int bf16, const float* mu, float* state, const int* slot_ids, const int* q_start,
                             const int* q_lens, const int* context_lens, void* out, int batch, int tokens, int width,
                             int mixes, void* stream) {
  if (batch <= 0 || tokens <= 0) return 0;
  if (width < 1 || mixes < 1 || mixes > kMaxMixes || tokens > 65535 * kMixTokens || (q_lens == nullptr && tokens != batch)) return -2;
  TokenMixParams p{h, mu, state, slot_ids, q_start, q_lens, context_lens, out, batch, tokens, width, mixes};
  const bool vec = width % (bf16 ? 8 : 4) == 0 && al(h, 16) && al(out, 16);
  const bool one = tokens <= 512;
  const int cols = 128 * (vec ? (bf16 ? 8 : 4) : 1);
  const dim3 grid((width + cols - 1) / cols, one ? tokens : (tokens + kMixTokens - 1) / kMixTokens), block(128);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  using bf = __nv_bfloat16;
  if (bf16) {
    if (vec) return one ? launch_pdl(token_mix_kernel<8, 1, bf>, grid, block, 0, s, p)
                        : launch_pdl(token_mix_kernel<8, kMixTokens, bf>, grid, block, 0, s, p);
    return one ? launch_pdl(token_mix_kernel<1, 1, bf>, grid, block, 0, s, p)
               : launch_pdl(token_mix_kernel<1, kMixTokens, bf>, grid, block, 0, s, p);
  }
  if (vec) return one ? launch_pdl(token_mix_kernel<4, 1, float>, grid, block, 0, s, p)
                      : launch_pdl(token_mix_kernel<4, kMixTokens, float>, grid, block, 0, s, p);
  return one ? launch_pdl(token_mix_kernel<1, 1, float>, grid, block, 0, s, p)
             : launch_pdl(token_mix_kernel<1, kMixTokens, float>, grid, block, 0, s, p);
}

extern "C" int nkb_gate_heads(const void* x, int x_bf16, long long ld_token, long long ld_head, const NkbProj* gate,
                              int head_gate, int gate_act, const float* norm_w, int norm_stride, float eps, float scale, void* out,
                              int out_bf16, long long out_ld, int tokens, int heads, int width, void* stream) {
  if (tokens <= 0) return 0;
  if (heads < 1 || width < 1 || gate_act < 0 || gate_act >= ACT_COUNT) return -2;
  GateHeadsParams p{x, ld_token, ld_head, *gate, norm_w, out, out_ld, (long long)tokens * heads, gate_act, norm_stride,
                    heads, width, head_gate, eps, scale};
  return launch_gate_heads(p, x_bf16, out_bf16, reinterpret_cast<cudaStream_t>(stream));
}
