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
//   scan   any number of new tokens per sequence.  A CTA owns some columns of one head of one sequence for all of its
//          tokens; sixteen lanes share a set of columns, each holding every sixteenth group of four channels of them in
//          registers, so a token costs one packed subtract and two packed multiply-adds per two state elements, and the
//          gates and queries read from shared memory serve all of a lane's columns.  Sixteen partial sums (tokens x
//          columns) are exchanged together: a transposing butterfly of fifteen shuffles leaves each of the sixteen
//          lanes with one finished value.  The next tile of tokens is fetched while the current one is multiplied.
//   step   one new token per sequence (decode).  A CTA owns a head of a sequence, streams its state through
//          registers once (the whole state of a 128 x 128 head is in flight at once), and applies the per-head
//          norm of the result itself.
#include "common.cuh"
#include "proj_src.cuh"
#include "api.h"
#include <type_traits>

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

// four consecutive channels of a token as fetched: bf16 values stay packed until they are needed
template <int V>
struct RawGroup {
  float4 v;
  __device__ __forceinline__ void clear() { v = make_float4(0.f, 0.f, 0.f, 0.f); }
  __device__ __forceinline__ float4 get() const { return v; }
};
constexpr int kPackedBf16 = 2;     // V of the packed form: aligned bf16 values
template <>
struct RawGroup<kPackedBf16> {
  uint2 v;
  __device__ __forceinline__ void clear() { v = make_uint2(0u, 0u); }
  __device__ __forceinline__ float4 get() const {
    const float2 a = unpack_bf16x2(v.x), b = unpack_bf16x2(v.y);
    return make_float4(a.x, a.y, b.x, b.y);
  }
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
template <int V>
__device__ __forceinline__ void fetch_group(RawGroup<V>& r, const NkbProj& s, long long row, int head_col, int c, int dim) {
  if constexpr (V == kPackedBf16)
    r.v = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(s.ptr) + row * s.ld + head_col + c);
  else
    r.v = load_group<V>(s, row, head_col, c, dim);
}
__device__ __forceinline__ float query_act(float u, bool on) { return on ? u * sigmoid_f(u) : 0.f; }
__device__ __forceinline__ float forget_gate(float z, float bias, float lower, bool on) {
  return on ? lower + (1.f - lower) * sigmoid_f(z + bias) : 1.f;
}

constexpr int kScanThreads = 128;
constexpr int kScanLanes = 16;     // lanes that share the columns of a half warp
constexpr int kScanTokens = 8;     // tokens per tile

__device__ __forceinline__ float2 fsub2(float2 a, float2 b) {
  uint64_t rd;
  asm("sub.f32x2 %0, %1, %2;" : "=l"(rd) : "l"(reinterpret_cast<uint64_t&>(a)), "l"(reinterpret_cast<uint64_t&>(b)));
  return reinterpret_cast<float2&>(rd);
}

// CL: channels per lane (dim <= 16 CL), NC: columns per lane
template <int CL, int NC, int V, typename OutT>
__global__ void __launch_bounds__(kScanThreads, CL <= 8 ? 4 : 1)
hgrn2_scan_kernel(const __grid_constant__ RecurrentParams p) {
  constexpr int TT = kScanTokens, DP = kScanLanes * CL, COLS = 8 * NC;   // COLS: columns of the CTA
  constexpr int NG = TT * DP / 4 / kScanThreads > 0 ? TT * DP / 4 / kScanThreads : 1;
  constexpr int NVG = TT * COLS / 4;                // groups of four values per tile
  constexpr int NV = (NVG + kScanThreads - 1) / kScanThreads;
  constexpr int TB = kScanLanes / NC;               // tokens whose sums are exchanged together
  __shared__ __align__(16) float qs[2][TT][DP];
  __shared__ __align__(16) float fs[2][TT][DP];
  __shared__ __align__(16) float2 vs[2][TT][COLS];  // every value twice, as a packed pair
  __shared__ float os[TT][COLS];
  const int head = blockIdx.y, b = blockIdx.z, col0 = blockIdx.x * COLS;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane & 15;
  const int cl0 = (warp * 2 + (lane >> 4)) * NC;    // first of this lane's columns within the CTA
  griddep_wait();
  griddep_launch();
  const int n = p.q_lens[b], ctx = p.context_lens[b];
  if (n <= 0 || ctx < n) return;
  const int row0 = p.q_start[b];
  const int slot = p.slot_ids ? p.slot_ids[b] : b;
  const bool fresh = ctx == n;
  float* st = p.state + (((long long)slot * p.heads + head) * p.vdim + col0 + cl0) * p.dim_p;

  // channels of this lane: groups of four, group j at (j * 16 + g) * 4
  float2 S[NC][CL / 2];
#pragma unroll
  for (int k = 0; k < NC; ++k)
#pragma unroll
    for (int j = 0; j < CL / 4; ++j) {
      const int c = (j * kScanLanes + g) * 4;
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!fresh && col0 + cl0 + k < p.vdim && c < p.dim_p)
        x = *reinterpret_cast<const float4*>(st + (long long)k * p.dim_p + c);
      S[k][2 * j] = make_float2(x.x, x.y);
      S[k][2 * j + 1] = make_float2(x.z, x.w);
    }

  RawGroup<V> rq[NG], rf[NG], rv[NV];
  const int hq = head * p.dim, hv = head * p.vdim;
  // a thread fetches the same four channels of several tokens
  constexpr int kTokStep = kScanThreads / (DP / 4);
  const int lc = (threadIdx.x % (DP / 4)) * 4, ltok = threadIdx.x / (DP / 4);
  float fb[4], fl[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    fb[e] = lc + e < p.dim ? p.f_bias[hq + lc + e] : 0.f;
    fl[e] = lc + e < p.dim ? p.lower[hq + lc + e] : 0.f;
  }
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < NG; ++i) {
      const int tok = ltok + i * kTokStep;
      rq[i].clear();
      rf[i].clear();
      if (tok < TT && t0 + tok < n && lc < p.dim) {
        fetch_group<V>(rq[i], p.q, row0 + t0 + tok, hq, lc, p.dim);
        fetch_group<V>(rf[i], p.f, row0 + t0 + tok, hq, lc, p.dim);
      }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int idx = threadIdx.x + i * kScanThreads, tok = idx / (COLS / 4), c = col0 + idx % (COLS / 4) * 4;
      rv[i].clear();
      if (idx < NVG && t0 + tok < n && c < p.vdim) fetch_group<V>(rv[i], p.v, row0 + t0 + tok, hv, c, p.vdim);
    }
  };
  // activations of the fetched tile into shared memory; a token past the end keeps the state (f = 1, q = 0)
  auto publish = [&](int buf, int t0) {
#pragma unroll
    for (int i = 0; i < NG; ++i) {
      const int tok = ltok + i * kTokStep;
      if (tok < TT) {
        const bool on = t0 + tok < n;
        const float4 u = rq[i].get(), z = rf[i].get();
        float4 q, f;
        q.x = query_act(u.x, on && lc < p.dim);
        q.y = query_act(u.y, on && lc + 1 < p.dim);
        q.z = query_act(u.z, on && lc + 2 < p.dim);
        q.w = query_act(u.w, on && lc + 3 < p.dim);
        f.x = forget_gate(z.x, fb[0], fl[0], on && lc < p.dim);
        f.y = forget_gate(z.y, fb[1], fl[1], on && lc + 1 < p.dim);
        f.z = forget_gate(z.z, fb[2], fl[2], on && lc + 2 < p.dim);
        f.w = forget_gate(z.w, fb[3], fl[3], on && lc + 3 < p.dim);
        *reinterpret_cast<float4*>(&qs[buf][tok][lc]) = q;
        *reinterpret_cast<float4*>(&fs[buf][tok][lc]) = f;
      }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int idx = threadIdx.x + i * kScanThreads;
      if (idx < NVG) {
        const float4 x = rv[i].get();
        float4* dst = reinterpret_cast<float4*>(&vs[buf][idx / (COLS / 4)][idx % (COLS / 4) * 4]);
        dst[0] = make_float4(x.x, x.x, x.y, x.y);
        dst[1] = make_float4(x.z, x.z, x.w, x.w);
      }
    }
  };
  fetch(0);
  publish(0, 0);
  __syncthreads();
  int buf = 0;
#pragma unroll 1
  for (int t0 = 0; t0 < n; t0 += TT, buf ^= 1) {
    const bool more = t0 + TT < n;
    if (more) fetch(t0 + TT);
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
#pragma unroll
        for (int k = 0; k < NC; ++k) {
          const float2 v2 = vs[buf][h + tt][cl0 + k];
          float2 o = make_float2(0.f, 0.f);
#pragma unroll
          for (int j = 0; j < CL / 2; ++j) {
            S[k][j] = ffma2(f2[j], fsub2(S[k][j], v2), v2);
            o = ffma2(q2[j], S[k][j], o);
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
    if (more) publish(buf ^ 1, t0 + TT);
    __syncthreads();
    OutT* out = reinterpret_cast<OutT*>(p.out);
#pragma unroll
    for (int i = 0; i < TT * COLS / kScanThreads; ++i) {
      const int idx = threadIdx.x + i * kScanThreads, tok = idx / COLS, c = col0 + idx % COLS;
      if (t0 + tok < n && c < p.vdim)
        out[(long long)(row0 + t0 + tok) * p.heads * p.vdim + hv + c] = cast_out<OutT>(os[tok][idx % COLS]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int k = 0; k < NC; ++k)
#pragma unroll
    for (int j = 0; j < CL / 4; ++j) {
      const int c = (j * kScanLanes + g) * 4;
      if (col0 + cl0 + k < p.vdim && c < p.dim_p)
        *reinterpret_cast<float4*>(st + (long long)k * p.dim_p + c) =
            make_float4(S[k][2 * j].x, S[k][2 * j].y, S[k][2 * j + 1].x, S[k][2 * j + 1].y);
    }
}

// x[t, h, :] / sqrt(mean(x[t, h, :]^2) + eps) * w, in place; one warp per (token, head)
template <typename T>
__global__ void __launch_bounds__(256) head_rmsnorm_kernel(T* __restrict__ x, const float* __restrict__ w, long long n,
                                                           int vdim, float eps) {
  griddep_wait();
  griddep_launch();
  const long long i = (blockIdx.x * 256ll + threadIdx.x) >> 5;
  const int lane = threadIdx.x & 31;
  if (i >= n) return;
  T* r = x + i * vdim;
  float ss = 0.f;
  for (int c = lane; c < vdim; c += 32) {
    const float v = cast_in<T>(r[c]);
    ss += v * v;
  }
  const float inv = 1.f / sqrtf(warp_sum(ss) / float(vdim) + eps);
  for (int c = lane; c < vdim; c += 32) r[c] = cast_out<T>(cast_in<T>(r[c]) * inv * w[c]);
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

template <int CL, int NC, int V>
static int launch_scan_nc(const RecurrentParams& p, int batch, int out_bf16, cudaStream_t s) {
  const dim3 grid((p.vdim + 8 * NC - 1) / (8 * NC), p.heads, batch);
  return out_bf16 ? launch_pdl(hgrn2_scan_kernel<CL, NC, V, __nv_bfloat16>, grid, dim3(kScanThreads), 0, s, p)
                  : launch_pdl(hgrn2_scan_kernel<CL, NC, V, float>, grid, dim3(kScanThreads), 0, s, p);
}
// More columns per lane mean fewer shared-memory reads per state element, fewer mean more CTAs: take the most columns
// that still give (nearly) every SM a CTA.
template <int CL, int V>
static int launch_scan(const RecurrentParams& p, int batch, int out_bf16, cudaStream_t s) {
  const auto ctas = [&](int cols) { return (long long)batch * p.heads * ((p.vdim + cols - 1) / cols); };
  if constexpr (CL <= 8)
    if (ctas(64) >= 120) return launch_scan_nc<CL, 8, V>(p, batch, out_bf16, s);
  if (ctas(32) >= 120) return launch_scan_nc<CL, 4, V>(p, batch, out_bf16, s);
  return launch_scan_nc<CL, 2, V>(p, batch, out_bf16, s);
}
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

extern "C" int nkb_hgrn2_scan(const NkbProj* q, const NkbProj* f, const NkbProj* v, const float* f_bias,
                              const float* lower, float* state, const int* slot_ids, const int* q_start,
                              const int* q_lens, const int* context_lens, void* out, int out_bf16, int batch, int tokens,
                              int heads, int dim, int vdim, const float* norm_w, float eps, void* stream) {
  if (batch <= 0 || tokens <= 0) return 0;
  if (batch > 65535 || heads > 65535) return -2;
  RecurrentParams p{};
  if (int rc = recurrent_params(p, q, f, v, f_bias, lower, state, slot_ids, context_lens, out, heads, dim, vdim)) return rc;
  p.q_start = q_start;
  p.q_lens = q_lens;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const bool vec = dim % 4 == 0 && vdim % 4 == 0 && proj_vec4_ok(*q) && proj_vec4_ok(*f) && proj_vec4_ok(*v);
  const int form = !vec ? 1 : (q->bf16 && f->bf16 && v->bf16 ? kPackedBf16 : 4);
  const auto scan = [&](auto cl) {
    constexpr int CL = decltype(cl)::value;
    return form == 1 ? launch_scan<CL, 1>(p, batch, out_bf16, s)
                     : (form == 4 ? launch_scan<CL, 4>(p, batch, out_bf16, s) : launch_scan<CL, kPackedBf16>(p, batch, out_bf16, s));
  };
  const int rc = dim <= 64 ? scan(std::integral_constant<int, 4>{})
                           : (dim <= 128 ? scan(std::integral_constant<int, 8>{}) : scan(std::integral_constant<int, 16>{}));
  if (rc || !norm_w) return rc;
  const long long rows = (long long)tokens * heads;
  const dim3 grid(unsigned((rows + 7) / 8));
  return out_bf16 ? launch_pdl(head_rmsnorm_kernel<__nv_bfloat16>, grid, dim3(256), 0, s,
                               reinterpret_cast<__nv_bfloat16*>(out), norm_w, rows, vdim, eps)
                  : launch_pdl(head_rmsnorm_kernel<float>, grid, dim3(256), 0, s, reinterpret_cast<float*>(out), norm_w,
                               rows, vdim, eps);
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
