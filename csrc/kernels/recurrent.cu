// Gated linear recurrence with a per-channel forget gate (HGRN2), state in fp32.
//
//   f = lower + (1 - lower) * sigmoid(z + bias)          z, u, v: projections of the token
//   S[c, j] <- f[c] * S[c, j] + (1 - f[c]) * v[j]         = f[c] * (S[c, j] - v[j]) + v[j]
//   o[j] = sum_c silu(u[c]) * S[c, j]
//
// per head, c over `dim` channels and j over `vdim` values.  The state of a sequence lives in its slot of a
// [slots, heads, vdim, dim_p] array (dim_p = dim rounded up to a multiple of 4, so that a column is a run of
// 16-byte pieces); a sequence whose first new token has position 0 starts from zero, whatever the slot held.
//
// Two kernels:
//   scan   any number of new tokens per sequence.  A kernel of its own turns the projections into fp32 queries, gates and
//          value differences once per head.  A CTA then owns some columns of one head of one sequence for all of its
//          tokens; sixteen lanes share a set of columns, each holding every sixteenth group of four channels of them in
//          registers, so a token costs two packed multiply-adds per two state elements, and the gates and queries read from
//          shared memory serve all of a lane's columns.  Sixteen partial sums (tokens x columns) are exchanged together: a
//          transposing butterfly of fifteen shuffles leaves each of the sixteen lanes with one finished value.  The next
//          tile of tokens is copied while the current one is multiplied.
//   step   one new token per sequence (decode).  A CTA owns a head of a sequence, streams its state through
//          registers once (the whole state of a 128 x 128 head is in flight at once), and applies the per-head
//          norm of the result itself.
#include "common.cuh"
#include "proj_src.cuh"
#include "api.h"

namespace nkb {

struct RecurrentParams {
  NkbProj q, f, v;
  const float* f_bias;        // [heads * dim]
  const float* lower;         // [heads * dim]
  float* state;               // [slots, heads, vdim, dim_p]
  const int* slot_ids;        // [batch] or nullptr (slot = batch index)
  const int* q_start;         // scan only
  const int* q_lens;          // scan only
  const int* context_lens;    // counts the new tokens; negative = inactive
  void* out;                  // [tokens, heads * vdim]
  const float* norm_w;        // step only: [vdim]
  float eps;
  int heads, dim, dim_p, vdim;
};

template <int V>
__device__ __forceinline__ float4 load_group(const NkbProj& s, long long row, int head_col, int c, int dim) {
  if constexpr (V == 4) return proj_load4(s, row, head_col + c);
  float4 r = make_float4(0.f, 0.f, 0.f, 0.f);
  if (c < dim) r.x = proj_load(s, row, head_col + c);
  if (c + 1 < dim) r.y = proj_load(s, row, head_col + c + 1);
  if (c + 2 < dim) r.z = proj_load(s, row, head_col + c + 2);
  if (c + 3 < dim) r.w = proj_load(s, row, head_col + c + 3);
  return r;
}
__device__ __forceinline__ float query_act(float u, bool on) { return on ? u * sigmoid_f(u) : 0.f; }
__device__ __forceinline__ float forget_gate(float z, float bias, float lower, bool on) {
  return on ? lower + (1.f - lower) * sigmoid_f(z + bias) : 1.f;
}

constexpr int kScanThreads = 128;
constexpr int kScanLanes = 16;     // lanes that share the columns of a half warp

// Per-token inputs of the scan in fp32, computed once per head instead of once per column slice:
//   q_act [tokens, heads, dp], f_act [tokens, heads, dp]   silu(u) and the forget gate; channels past dim: 0 and 1
//   dv    [tokens, heads, vp]                              v_t - v_(t+1), with v_(t+1) = 0 for a sequence's last new token
template <int V>
__global__ void __launch_bounds__(256)
hgrn2_gates_kernel(const __grid_constant__ RecurrentParams p, float* __restrict__ q_act, float* __restrict__ f_act,
                   float* __restrict__ dv, int dp, int vp, int batch) {
  griddep_wait();
  griddep_launch();
  const long long t = blockIdx.x;
  bool end = false;
  for (int b = threadIdx.x; b < batch; b += blockDim.x) end = end || (t == (long long)p.q_start[b] + p.q_lens[b] - 1);
  const bool last = __syncthreads_or(end) != 0 || blockIdx.x + 1 == gridDim.x;
  const int gq = dp / 4, gv = vp / 4;
  for (int i = threadIdx.x; i < p.heads * gq; i += blockDim.x) {
    const int head = i / gq, c = (i % gq) * 4, hq = head * p.dim;
    float4 u = make_float4(0.f, 0.f, 0.f, 0.f), z = u;
    if (c < p.dim) {
      u = load_group<V>(p.q, t, hq, c, p.dim);
      z = load_group<V>(p.f, t, hq, c, p.dim);
    }
    const float uv[4] = {u.x, u.y, u.z, u.w}, zv[4] = {z.x, z.y, z.z, z.w};
    float qo[4], fo[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const bool on = c + e < p.dim;
      qo[e] = query_act(uv[e], on);
      fo[e] = on ? forget_gate(zv[e], p.f_bias[hq + c + e], p.lower[hq + c + e], true) : 1.f;
    }
    const long long o = (t * p.heads + head) * dp + c;
    *reinterpret_cast<float4*>(q_act + o) = make_float4(qo[0], qo[1], qo[2], qo[3]);
    *reinterpret_cast<float4*>(f_act + o) = make_float4(fo[0], fo[1], fo[2], fo[3]);
  }
  for (int i = threadIdx.x; i < p.heads * gv; i += blockDim.x) {
    const int head = i / gv, c = (i % gv) * 4, hv = head * p.vdim;
    float4 x = load_group<V>(p.v, t, hv, c, p.vdim);
    if (!last) {
      const float4 y = load_group<V>(p.v, t + 1, hv, c, p.vdim);
      x = make_float4(x.x - y.x, x.y - y.y, x.z - y.z, x.w - y.w);
    }
    *reinterpret_cast<float4*>(dv + (t * p.heads + head) * vp + c) = x;
  }
}

// 16 bytes global -> shared, zeros when `on` is false
__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool on) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(on ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// CL: channels per lane (dim <= 16 CL), NC: columns per lane.  The registers hold D = S - v of the next token, which
// takes one multiply-add per element and token (D <- f D + dv) where S takes two operations; v's share of the output,
// v_(t+1) sum(q), is added when the output is written, and D of a sequence's last new token is its state.
template <int CL, int NC, typename OutT>
__global__ void __launch_bounds__(kScanThreads, CL <= 8 ? 4 : 1)
hgrn2_scan_kernel(const __grid_constant__ RecurrentParams p, const float* __restrict__ q_act,
                  const float* __restrict__ f_act, const float* __restrict__ dv, int vp) {
  constexpr int TT = CL <= 8 ? 16 : 8;              // tokens per tile
  constexpr int DP = kScanLanes * CL, COLS = 8 * NC;
  constexpr int TB = kScanLanes / NC;               // tokens whose sums are exchanged together
  constexpr int NO = TT * COLS / kScanThreads;      // outputs of a thread per tile
  __shared__ __align__(16) float qs[2][TT][DP];
  __shared__ __align__(16) float fs[2][TT][DP];
  __shared__ __align__(16) float ds[2][TT][COLS];
  __shared__ float os[TT][COLS];
  __shared__ float qsum[TT];
  const int head = blockIdx.y, b = blockIdx.z, col0 = blockIdx.x * COLS;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane & 15;
  const int cl0 = (warp * 2 + (lane >> 4)) * NC;    // first of this lane's columns within the CTA
  griddep_wait();
  griddep_launch();
  const int n = p.q_lens[b], ctx = p.context_lens[b];
  if (n <= 0 || ctx < n) return;
  const long long row0 = p.q_start[b];
  const int slot = p.slot_ids ? p.slot_ids[b] : b;
  const bool fresh = ctx == n;
  const int hv = head * p.vdim;
  float* st = p.state + (((long long)slot * p.heads + head) * p.vdim + col0 + cl0) * p.dim_p;

  auto fetch = [&](int buf, int t0) {
#pragma unroll
    for (int i = 0; i < TT * DP / 4 / kScanThreads; ++i) {
      const int idx = threadIdx.x + i * kScanThreads, tok = idx / (DP / 4), c = idx % (DP / 4) * 4;
      const bool on = t0 + tok < n;
      const long long o = ((row0 + (on ? t0 + tok : 0)) * p.heads + head) * DP + c;
      cp_async16(&qs[buf][tok][c], q_act + o, on);
      cp_async16(&fs[buf][tok][c], f_act + o, on);
    }
#pragma unroll
    for (int i = 0; i < (TT * COLS / 4 + kScanThreads - 1) / kScanThreads; ++i) {
      const int idx = threadIdx.x + i * kScanThreads, tok = idx / (COLS / 4), c = idx % (COLS / 4) * 4;
      if (idx < TT * COLS / 4) {
        const bool on = t0 + tok < n && col0 + c < vp;
        const long long o = on ? ((row0 + t0 + tok) * p.heads + head) * vp + col0 + c : 0;
        cp_async16(&ds[buf][tok][c], dv + o, on);
      }
    }
    cp_async_commit();
  };
  fetch(0, 0);

  // channels of this lane: groups of four, group j at (j * 16 + g) * 4
  float2 D[NC][CL / 2];
#pragma unroll
  for (int k = 0; k < NC; ++k) {
    const bool ok = col0 + cl0 + k < p.vdim;
    const float v0 = ok ? proj_load(p.v, row0, hv + col0 + cl0 + k) : 0.f;
#pragma unroll
    for (int j = 0; j < CL / 4; ++j) {
      const int c = (j * kScanLanes + g) * 4;
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!fresh && ok && c < p.dim_p) x = *reinterpret_cast<const float4*>(st + (long long)k * p.dim_p + c);
      D[k][2 * j] = make_float2(x.x - v0, x.y - v0);
      D[k][2 * j + 1] = make_float2(x.z - v0, x.w - v0);
    }
  }

  int buf = 0;
#pragma unroll 1
  for (int t0 = 0; t0 < n; t0 += TT, buf ^= 1) {
    cp_async_wait_all();
    __syncthreads();                                 // the tile is there; nobody reads the other buffer or os any more
    if (t0 + TT < n) {
      fetch(buf ^ 1, t0 + TT);
    } else {
      // tokens past the end keep D: gate one (query and dv are zero-filled)
      for (int i = threadIdx.x; i < (t0 + TT - n) * DP; i += kScanThreads) fs[buf][n - t0 + i / DP][i % DP] = 1.f;
      __syncthreads();
    }
    // v of the token after each of this thread's outputs, as fetched: a conversion here would wait for the load
    uint32_t vn[NO];
#pragma unroll
    for (int i = 0; i < NO; ++i) {
      const int idx = threadIdx.x + i * kScanThreads, tok = idx / COLS, c = col0 + idx % COLS;
      vn[i] = 0u;
      if (t0 + tok + 1 < n && c < p.vdim) {
        const long long r = row0 + t0 + tok + 1;
        if (p.v.bf16)
          vn[i] = reinterpret_cast<const uint16_t*>(p.v.ptr)[r * p.v.ld + hv + c];
        else
          vn[i] = __float_as_uint(proj_load(p.v, r, hv + c));
      }
    }
#pragma unroll
    for (int tok = warp; tok < TT; tok += kScanThreads / 32) {
      float a = 0.f;
#pragma unroll
      for (int i = 0; i < DP / 32; ++i) a += qs[buf][tok][lane + 32 * i];
      a = warp_sum(a);
      if (lane == 0) qsum[tok] = a;
    }
#pragma unroll 1
    for (int h = 0; h < TT; h += TB) {
      if (t0 + h >= n) break;
      float po[kScanLanes];                          // [token][column]
#pragma unroll
      for (int tt = 0; tt < TB; ++tt) {
        float2 f2[CL / 2], q2[CL / 2];
#pragma unroll
        for (int j = 0; j < CL / 4; ++j) {
          const float4 f = *reinterpret_cast<const float4*>(&fs[buf][h + tt][(j * kScanLanes + g) * 4]);
          const float4 q = *reinterpret_cast<const float4*>(&qs[buf][h + tt][(j * kScanLanes + g) * 4]);
          f2[2 * j] = make_float2(f.x, f.y); f2[2 * j + 1] = make_float2(f.z, f.w);
          q2[2 * j] = make_float2(q.x, q.y); q2[2 * j + 1] = make_float2(q.z, q.w);
        }
        float d[NC];
        if constexpr (NC >= 4) {
#pragma unroll
          for (int k = 0; k < NC; k += 4) {
            const float4 x = *reinterpret_cast<const float4*>(&ds[buf][h + tt][cl0 + k]);
            d[k] = x.x; d[k + 1] = x.y; d[k + 2] = x.z; d[k + 3] = x.w;
          }
        } else {
#pragma unroll
          for (int k = 0; k < NC; ++k) d[k] = ds[buf][h + tt][cl0 + k];
        }
#pragma unroll
        for (int k = 0; k < NC; ++k) {
          const float2 d2 = make_float2(d[k], d[k]);
          float2 o = make_float2(0.f, 0.f);
#pragma unroll
          for (int j = 0; j < CL / 2; ++j) {
            D[k][j] = ffma2(f2[j], D[k][j], d2);
            o = ffma2(q2[j], D[k][j], o);
          }
          po[tt * NC + k] = o.x + o.y;
        }
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
    OutT* out = reinterpret_cast<OutT*>(p.out);
#pragma unroll
    for (int i = 0; i < NO; ++i) {
      const int idx = threadIdx.x + i * kScanThreads, tok = idx / COLS, c = col0 + idx % COLS;
      if (t0 + tok < n && c < p.vdim)
        out[(row0 + t0 + tok) * p.heads * p.vdim + hv + c] = cast_out<OutT>(
            fmaf(__uint_as_float(p.v.bf16 ? vn[i] << 16 : vn[i]), qsum[tok], os[tok][idx % COLS]));
    }
  }
#pragma unroll
  for (int k = 0; k < NC; ++k)
#pragma unroll
    for (int j = 0; j < CL / 4; ++j) {
      const int c = (j * kScanLanes + g) * 4;
      if (col0 + cl0 + k < p.vdim && c < p.dim_p)
        *reinterpret_cast<float4*>(st + (long long)k * p.dim_p + c) =
            make_float4(D[k][2 * j].x, D[k][2 * j].y, D[k][2 * j + 1].x, D[k][2 * j + 1].y);
    }
}

// x[t, h, :] / sqrt(mean(x[t, h, :]^2) + eps) * w, in place; one warp per (token, head).  VEC: vdim is a multiple of 4
// and at most 128, so that a lane holds its four elements in registers.
template <bool VEC, typename T>
__global__ void __launch_bounds__(256) head_rmsnorm_kernel(T* __restrict__ x, const float* __restrict__ w, long long n,
                                                           int vdim, float eps) {
  griddep_wait();
  griddep_launch();
  const long long i = (blockIdx.x * 256ll + threadIdx.x) >> 5;
  const int lane = threadIdx.x & 31;
  if (i >= n) return;
  T* r = x + i * vdim;
  if constexpr (VEC) {
    const int c = lane * 4;
    const bool on = c < vdim;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (on) {
      if constexpr (sizeof(T) == 2) {
        const uint2 u = *reinterpret_cast<const uint2*>(r + c);
        const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
        v = make_float4(a.x, a.y, b.x, b.y);
      } else {
        v = *reinterpret_cast<const float4*>(r + c);
      }
    }
    const float ss = warp_sum(v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w);
    const float inv = 1.f / sqrtf(ss / float(vdim) + eps);
    if (on) {
      const float4 ww = *reinterpret_cast<const float4*>(w + c);
      v = make_float4(v.x * inv * ww.x, v.y * inv * ww.y, v.z * inv * ww.z, v.w * inv * ww.w);
      if constexpr (sizeof(T) == 2)
        *reinterpret_cast<uint2*>(r + c) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
      else
        *reinterpret_cast<float4*>(r + c) = v;
    }
    return;
  }
  float ss = 0.f;
  for (int c = lane; c < vdim; c += 32) {
    const float v = cast_in<T>(r[c]);
    ss += v * v;
  }
  const float inv = 1.f / sqrtf(warp_sum(ss) / float(vdim) + eps);
  for (int c = lane; c < vdim; c += 32) r[c] = cast_out<T>(cast_in<T>(r[c]) * inv * w[c]);
}
template <typename T>
static int launch_head_rmsnorm(void* x, const float* w, long long rows, int vdim, float eps, cudaStream_t s) {
  const bool vec = vdim % 4 == 0 && vdim <= 128 && ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w)) & 15) == 0;
  const dim3 grid(unsigned((rows + 7) / 8));
  return vec ? launch_pdl(head_rmsnorm_kernel<true, T>, grid, dim3(256), 0, s, reinterpret_cast<T*>(x), w, rows, vdim, eps)
             : launch_pdl(head_rmsnorm_kernel<false, T>, grid, dim3(256), 0, s, reinterpret_cast<T*>(x), w, rows, vdim, eps);
}

constexpr int kStepThreads = 256;
constexpr int kStepBlocks = 4;      // column blocks of 32 in flight

template <int CH, typename OutT>
__global__ void __launch_bounds__(kStepThreads)
hgrn2_step_kernel(const __grid_constant__ RecurrentParams p) {
  constexpr int D8 = 8 * CH;
  __shared__ __align__(16) float qs[D8];
  __shared__ __align__(16) float fs[D8];
  __shared__ float red[kStepThreads / 32];
  extern __shared__ float dyn[];                    // v [vdim], o [vdim]
  float* vs = dyn;
  float* os = dyn + p.vdim;
  const int head = blockIdx.x, b = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane & 7;
  const int cl = warp * 4 + (lane >> 3);
  griddep_wait();
  griddep_launch();
  OutT* out = reinterpret_cast<OutT*>(p.out) + ((long long)b * p.heads + head) * p.vdim;
  const int ctx = p.context_lens[b];
  if (ctx <= 0) {
    for (int c = threadIdx.x; c < p.vdim; c += kStepThreads) out[c] = cast_out<OutT>(0.f);
    return;
  }
  const int slot = p.slot_ids ? p.slot_ids[b] : b;
  const bool fresh = ctx == 1;
  float* st = p.state + ((long long)slot * p.heads + head) * p.vdim * p.dim_p;
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
        if (!fresh && col < p.vdim && c < p.dim_p)
          S[k][j] = __ldcs(reinterpret_cast<const float4*>(st + (long long)col * p.dim_p + c));
      }
    }
    if (b0 == 0) {
      for (int c = threadIdx.x; c < D8; c += kStepThreads) {
        const bool on = c < p.dim;
        qs[c] = query_act(on ? proj_load(p.q, b, head * p.dim + c) : 0.f, on);
        fs[c] = on ? forget_gate(proj_load(p.f, b, head * p.dim + c), p.f_bias[head * p.dim + c],
                                 p.lower[head * p.dim + c], true)
                   : 1.f;
      }
      for (int c = threadIdx.x; c < p.vdim; c += kStepThreads) vs[c] = proj_load(p.v, b, head * p.vdim + c);
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
        const float4 f = *reinterpret_cast<const float4*>(&fs[c]);
        const float4 q = *reinterpret_cast<const float4*>(&qs[c]);
        float4 s = S[k][j];
        s.x = fmaf(f.x, s.x - v, v);
        s.y = fmaf(f.y, s.y - v, v);
        s.z = fmaf(f.z, s.z - v, v);
        s.w = fmaf(f.w, s.w - v, v);
        o = fmaf(q.x, s.x, o);
        o = fmaf(q.y, s.y, o);
        o = fmaf(q.z, s.z, o);
        o = fmaf(q.w, s.w, o);
        if (ok && c < p.dim_p) __stcs(reinterpret_cast<float4*>(st + (long long)col * p.dim_p + c), s);
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
  const float inv = 1.f / sqrtf(tot / float(p.vdim) + p.eps);
  for (int c = threadIdx.x; c < p.vdim; c += kStepThreads) out[c] = cast_out<OutT>(os[c] * inv * p.norm_w[c]);
}

struct ScanInputs {
  const float *q_act, *f_act, *dv;
  int vp;
};
template <int CL, int NC>
static int launch_scan_nc(const RecurrentParams& p, const ScanInputs& in, int batch, int out_bf16, cudaStream_t s) {
  const dim3 grid((p.vdim + 8 * NC - 1) / (8 * NC), p.heads, batch);
  return out_bf16 ? launch_pdl(hgrn2_scan_kernel<CL, NC, __nv_bfloat16>, grid, dim3(kScanThreads), 0, s, p, in.q_act,
                               in.f_act, in.dv, in.vp)
                  : launch_pdl(hgrn2_scan_kernel<CL, NC, float>, grid, dim3(kScanThreads), 0, s, p, in.q_act, in.f_act,
                               in.dv, in.vp);
}
// More columns per lane mean fewer shared-memory reads per state element, fewer mean more warps to hide latency with:
// eight columns from about two CTAs per SM on, two when even four would leave SMs with a single CTA (measured on one,
// two, four and eight sequences of 32 heads of 128 x 128).
template <int CL>
static int launch_scan(const RecurrentParams& p, const ScanInputs& in, int batch, int out_bf16, cudaStream_t s) {
  const auto ctas = [&](int cols) { return (long long)batch * p.heads * ((p.vdim + cols - 1) / cols); };
  if constexpr (CL <= 8)
    if (ctas(64) >= 2 * 148) return launch_scan_nc<CL, 8>(p, in, batch, out_bf16, s);
  if (ctas(32) >= 200) return launch_scan_nc<CL, 4>(p, in, batch, out_bf16, s);
  return launch_scan_nc<CL, 2>(p, in, batch, out_bf16, s);
}
static int scan_channels(int dim) { return dim <= 64 ? 64 : (dim <= 128 ? 128 : 256); }
template <int CH>
static int launch_step(const RecurrentParams& p, int batch, int out_bf16, cudaStream_t s) {
  const dim3 grid(p.heads, batch);
  const size_t smem = size_t(2 * p.vdim) * sizeof(float);
  return out_bf16 ? launch_pdl(hgrn2_step_kernel<CH, __nv_bfloat16>, grid, dim3(kStepThreads), smem, s, p)
                  : launch_pdl(hgrn2_step_kernel<CH, float>, grid, dim3(kStepThreads), smem, s, p);
}

}  // namespace nkb

using namespace nkb;

static int recurrent_params(RecurrentParams& p, const NkbProj* q, const NkbProj* f, const NkbProj* v,
                            const float* f_bias, const float* lower, float* state, const int* slot_ids,
                            const int* context_lens, void* out, int heads, int dim, int vdim) {
  if (heads < 1 || dim < 1 || dim > 256 || vdim < 1 || vdim > 1024 || !state || !context_lens) return -2;
  p.q = *q; p.f = *f; p.v = *v;
  p.f_bias = f_bias; p.lower = lower; p.state = state; p.slot_ids = slot_ids; p.context_lens = context_lens;
  p.out = out; p.heads = heads; p.dim = dim; p.dim_p = (dim + 3) / 4 * 4; p.vdim = vdim;
  return 0;
}

// floats of scratch one token of a scan needs
extern "C" long long nkb_hgrn2_scan_scratch(int heads, int dim, int vdim) {
  return (long long)heads * (2 * scan_channels(dim) + (vdim + 3) / 4 * 4);
}

// scratch: tokens * nkb_hgrn2_scan_scratch(...) floats, 16-byte aligned.  Every row of the packed batch belongs to one
// of the sequences.
extern "C" int nkb_hgrn2_scan(const NkbProj* q, const NkbProj* f, const NkbProj* v, const float* f_bias,
                              const float* lower, float* state, const int* slot_ids, const int* q_start,
                              const int* q_lens, const int* context_lens, float* scratch, void* out, int out_bf16,
                              int batch, int tokens, int heads, int dim, int vdim, const float* norm_w, float eps,
                              void* stream) {
  if (batch <= 0 || tokens <= 0) return 0;
  if (batch > 65535 || heads > 65535 || !scratch || (reinterpret_cast<uintptr_t>(scratch) & 15)) return -2;
  RecurrentParams p{};
  if (int rc = recurrent_params(p, q, f, v, f_bias, lower, state, slot_ids, context_lens, out, heads, dim, vdim)) return rc;
  p.q_start = q_start;
  p.q_lens = q_lens;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const bool vec = dim % 4 == 0 && vdim % 4 == 0 && proj_vec4_ok(*q) && proj_vec4_ok(*f) && proj_vec4_ok(*v);
  const int dp = scan_channels(dim), vp = (vdim + 3) / 4 * 4;
  float* q_act = scratch;
  float* f_act = q_act + (long long)tokens * heads * dp;
  float* dv = f_act + (long long)tokens * heads * dp;
  int rc = vec ? launch_pdl(hgrn2_gates_kernel<4>, dim3(tokens), dim3(256), 0, s, p, q_act, f_act, dv, dp, vp, batch)
               : launch_pdl(hgrn2_gates_kernel<1>, dim3(tokens), dim3(256), 0, s, p, q_act, f_act, dv, dp, vp, batch);
  if (rc) return rc;
  const ScanInputs in{q_act, f_act, dv, vp};
  rc = dp == 64 ? launch_scan<4>(p, in, batch, out_bf16, s)
                : (dp == 128 ? launch_scan<8>(p, in, batch, out_bf16, s) : launch_scan<16>(p, in, batch, out_bf16, s));
  if (rc || !norm_w) return rc;
  const long long rows = (long long)tokens * heads;
  return out_bf16 ? launch_head_rmsnorm<__nv_bfloat16>(out, norm_w, rows, vdim, eps, s)
                  : launch_head_rmsnorm<float>(out, norm_w, rows, vdim, eps, s);
}

extern "C" int nkb_hgrn2_step(const NkbProj* q, const NkbProj* f, const NkbProj* v, const float* f_bias,
                              const float* lower, float* state, const int* slot_ids, const int* context_lens, void* out,
                              int out_bf16, int batch, int heads, int dim, int vdim, const float* norm_w, float eps,
                              void* stream) {
  if (batch <= 0) return 0;
  if (batch > 65535 || !norm_w) return -2;
  RecurrentParams p{};
  if (int rc = recurrent_params(p, q, f, v, f_bias, lower, state, slot_ids, context_lens, out, heads, dim, vdim)) return rc;
  p.norm_w = norm_w;
  p.eps = eps;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (dim <= 32) return launch_step<4>(p, batch, out_bf16, s);
  if (dim <= 64) return launch_step<8>(p, batch, out_bf16, s);
  if (dim <= 128) return launch_step<16>(p, batch, out_bf16, s);
  return launch_step<32>(p, batch, out_bf16, s);
}
