// Mixers whose heads carry a matrix state: gated delta rule, bonus recurrence, normalised matrix memory.
//   chunk path   short convolution + SiLU + unit vectors (or mixes with the previous token), the recurrence over the chunk's rows,
//                read-out norm and gate
//   one token    one kernel: unit vectors, low-rank decay and gate, state update, read-out, norm and gate
//
// A value column of S evolves on its own given q, k and the decay, so columns are spread over the GPU and the tokens of a chunk run
// one after the other, all in fp32 (packed pairs): eight lanes share a column, lane l holds the 16-byte pieces l, l + 8, ... of
// its dim entries in registers for the whole chunk.  Rows arrive in shared memory tile by tile through cp.async, two tiles deep.
#include "stack.cuh"
#include "launch.hpp"

#include <string.h>

using namespace nrt;

namespace {

typedef unsigned long long u64;
constexpr int kLanes = 8;                     // lanes per value column
constexpr float kUnitEps = 1e-6f;             // unit vectors: x / sqrt(sum(x^2) + 1e-6)

__device__ __forceinline__ u64 pack2(float x, float y) {
  u64 v;
  asm("mov.b64 %0, {%1, %2};" : "=l"(v) : "f"(x), "f"(y));
  return v;
}
__device__ __forceinline__ u64 fma2(u64 a, u64 b, u64 c) {
  u64 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ u64 mul2(u64 a, u64 b) {
  u64 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ float both(u64 a) {
  float x, y;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(a));
  return x + y;
}
__device__ __forceinline__ float column_sum(float v) {                 // over the eight lanes of a column
  v += __shfl_xor_sync(0xffffffffu, v, 1);
  v += __shfl_xor_sync(0xffffffffu, v, 2);
  v += __shfl_xor_sync(0xffffffffu, v, 4);
  return v;
}
__device__ __forceinline__ void cp_async(float* dst, const float* src, bool vec) {
  if (vec) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
  else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ bool quads(const float* p, long long ld, int n) {      // rows of n floats reachable in 16-byte pieces
  return ((reinterpret_cast<uintptr_t>(p) & 15) | (uintptr_t)((ld | n) & 3)) == 0;
}
// Rows [0, n) of `cols` floats into shared rows of `pitch`.
__device__ __forceinline__ void stage_rows(float* dst, int pitch, const float* src, long long ld, int n, int cols, bool vec) {
  const int step = vec ? 4 : 1, per = cols / step;
  for (int i = threadIdx.x; i < n * per; i += blockDim.x) {
    const int t = i / per, c = (i - t * per) * step;
    cp_async(dst + t * pitch + c, src + t * ld + c, vec);
  }
}

__host__ __device__ inline int pad4(int n) { return (n + 3) / 4 * 4; }
template <int KIND>
__host__ __device__ constexpr int extra_columns() { return KIND == kStateNormalized ? 1 : 0; }      // the normaliser is a column with v = 1

// One token of one column: state in `s`, this lane's pieces of q, k (and g) in shared memory.  Returns the read-out's partial sum.
template <int KIND, int NV>
__device__ __forceinline__ float column_step(u64 (&s)[2 * NV], const ulonglong2* q, const ulonglong2* k, const ulonglong2* g, float v,
                                             float s0, float s1) {
  u64 a0 = 0ull, a1 = 0ull;
  if (KIND == kStateDelta) {                   // s0 = step size
    ulonglong2 kk[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const ulonglong2 gg = g[i * kLanes];
      kk[i] = k[i * kLanes];
      s[2 * i] = mul2(s[2 * i], gg.x);
      s[2 * i + 1] = mul2(s[2 * i + 1], gg.y);
      a0 = fma2(s[2 * i], kk[i].x, a0);
      a1 = fma2(s[2 * i + 1], kk[i].y, a1);
    }
    const float u = s0 * (v - column_sum(both(a0) + both(a1)));
    const u64 uu = pack2(u, u);
    a0 = a1 = 0ull;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const ulonglong2 qq = q[i * kLanes];
      s[2 * i] = fma2(kk[i].x, uu, s[2 * i]);
      s[2 * i + 1] = fma2(kk[i].y, uu, s[2 * i + 1]);
      a0 = fma2(s[2 * i], qq.x, a0);
      a1 = fma2(s[2 * i + 1], qq.y, a1);
    }
    return both(a0) + both(a1);
  }
  if (KIND == kStateBonus) {
    const u64 vv = pack2(v, v);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const ulonglong2 qq = q[i * kLanes], kk = k[i * kLanes], gg = g[i * kLanes];
      a0 = fma2(s[2 * i], qq.x, a0);
      a1 = fma2(s[2 * i + 1], qq.y, a1);
      s[2 * i] = fma2(s[2 * i], gg.x, mul2(kk.x, vv));
      s[2 * i + 1] = fma2(s[2 * i + 1], gg.y, mul2(kk.y, vv));
    }
    return both(a0) + both(a1);
  }
  const float b = s1 * v;                      // s0, s1 = what is kept, what is added
  const u64 aa = pack2(s0, s0), bb = pack2(b, b);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const ulonglong2 qq = q[i * kLanes], kk = k[i * kLanes];
    s[2 * i] = fma2(s[2 * i], aa, mul2(kk.x, bb));
    s[2 * i + 1] = fma2(s[2 * i + 1], aa, mul2(kk.y, bb));
    a0 = fma2(s[2 * i], qq.x, a0);
    a1 = fma2(s[2 * i + 1], qq.y, a1);
  }
  return both(a0) + both(a1);
}

// Log gates of the normalised form.
__device__ __forceinline__ float log_input(float z, float cap) { return soft_cap(z, cap); }
__device__ __forceinline__ float log_forget(float z, float cap) { return -softplus_f(-soft_cap(z, cap)); }

// ------------------------------------------------------------------------------------ chunk path: the recurrence
// grid (column tiles, heads); a warp holds four columns.
__host__ __device__ inline int chunk_stage_floats(int kind, int dp, int cols, int tokens) {
  return tokens * ((kind == kStateNormalized ? 2 : 3) * dp + cols + 4);
}

template <int KIND, int NV>
__global__ void __launch_bounds__(256) state_chunk_kernel(const StateChunkArgs a, const int tokens) {
  constexpr int DP = NV * 4 * kLanes;
  extern __shared__ __align__(16) float sh[];
  griddep_wait();
  griddep_launch();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, l = lane & (kLanes - 1);
  const int cols = (blockDim.x >> 5) * 4, C = a.vdim + extra_columns<KIND>(), d4 = pad4(a.dim);
  const int h = blockIdx.y, hk = h / (a.heads / a.kv_heads), c0 = blockIdx.x * cols, c = c0 + warp * 4 + lane / kLanes;
  const int pos0 = *a.pos0;
  const int slot = state_slot(a.tags, pos0, a.status);
  if (slot < 0) return;
  const float* old = a.state + slot * a.state_stride;
  float* now = a.state + (1 - slot) * a.state_stride;
  const long long at = ((long long)h * C + c) * d4;
  const bool live = c < C;

  u64 s[2 * NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    ulonglong2 v = make_ulonglong2(0ull, 0ull);
    const int e = (l + kLanes * i) * 4;
    if (live && pos0 > 0 && e < d4) v = *reinterpret_cast<const ulonglong2*>(old + at + e);
    s[2 * i] = v.x;
    s[2 * i + 1] = v.y;
  }
  float m = KIND == kStateNormalized && pos0 > 0 ? old[(long long)a.heads * C * d4 + h] : 0.f;

  const int stage = chunk_stage_floats(KIND, DP, cols, tokens);
  for (int i = threadIdx.x; i < 2 * stage; i += blockDim.x) sh[i] = 0.f;      // columns beyond dim stay zero
  __syncthreads();
  const float* q0 = a.q + (long long)hk * a.dim;
  const float* k0 = a.k + (long long)hk * a.dim;
  const float* g0 = KIND == kStateNormalized ? nullptr : a.g + (long long)h * a.dim;
  const float* v0 = a.v + (long long)h * a.vdim + c0;
  const int vcols = min(cols, a.vdim - c0);                              // (none in a tile that holds only the normaliser)
  const bool qv = quads(q0, a.q_ld, a.dim), kv = quads(k0, a.k_ld, a.dim), gv = KIND != kStateNormalized && quads(g0, a.g_ld, a.dim),
             vv = vcols > 0 && quads(v0, a.v_ld, vcols);
  auto parts = [&](int st, float*& sk, float*& sq, float*& sg, float*& sv, float*& sc) {
    sk = sh + st * stage;
    sq = sk + tokens * DP;
    sg = sq + tokens * DP;
    sv = KIND == kStateNormalized ? sg : sg + tokens * DP;
    sc = sv + tokens * cols;                                             // four scalars per token: two raw, two derived
  };
  auto request = [&](int r0, int st) {
    const int n = min(tokens, a.rows - r0);
    float *sk, *sq, *sg, *sv, *sc;
    parts(st, sk, sq, sg, sv, sc);
    stage_rows(sk, DP, k0 + r0 * a.k_ld, a.k_ld, n, a.dim, kv);
    stage_rows(sq, DP, q0 + r0 * a.q_ld, a.q_ld, n, a.dim, qv);
    if (KIND != kStateNormalized) stage_rows(sg, DP, g0 + r0 * a.g_ld, a.g_ld, n, a.dim, gv);
    if (vcols > 0) stage_rows(sv, cols, v0 + r0 * a.v_ld, a.v_ld, n, vcols, vv);
    if (KIND == kStateDelta) stage_rows(sc, 4, a.beta + r0 * a.beta_ld + h, a.beta_ld, n, 1, false);
    if (KIND == kStateNormalized) {
      stage_rows(sc, 4, a.gi + r0 * a.gate_ld + h, a.gate_ld, n, 1, false);
      stage_rows(sc + 1, 4, a.gf + r0 * a.gate_ld + h, a.gate_ld, n, 1, false);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  request(0, 0);
  int st = 0;
  for (int r0 = 0; r0 < a.rows; r0 += tokens, st ^= 1) {
    const int n = min(tokens, a.rows - r0);
    if (r0 + tokens < a.rows) {
      request(r0 + tokens, st ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    float *sk, *sq, *sg, *sv, *sc;
    parts(st, sk, sq, sg, sv, sc);
    // scalars of the tile's tokens
    if (KIND == kStateDelta) {
      if ((int)threadIdx.x < n) sc[threadIdx.x * 4 + 2] = sigmoid_f(sc[threadIdx.x * 4]);
    } else if (KIND == kStateBonus) {
      for (int t = warp; t < n; t += blockDim.x >> 5) {
        float b = 0.f;
        for (int d = lane; d < a.dim; d += 32) b = fmaf(sq[t * DP + d] * bf(a.u + (long long)h * a.dim + d), sk[t * DP + d], b);
        b = lane_sum(b);
        if (lane == 0) sc[t * 4 + 2] = b;
      }
    } else if (warp == 0) {
      // running maximum over the tile: m -> max(f + m, i) composes as (sum of f, max), scanned over the lanes
      const float zi = lane < n ? log_input(sc[lane * 4], a.cap) : 0.f, zf = lane < n ? log_forget(sc[lane * 4 + 1], a.cap) : 0.f;
      float f = zf, b = lane < n ? zi : -FLT_MAX;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float fp = __shfl_up_sync(0xffffffffu, f, o), bp = __shfl_up_sync(0xffffffffu, b, o);
        if (lane >= o) {
          b = fmaxf(f + bp, b);
          f += fp;
        }
      }
      const float mt = fmaxf(f + m, b);
      float before = __shfl_up_sync(0xffffffffu, mt, 1);
      if (lane == 0) before = m;
      if (lane < n) {
        sc[lane * 4] = expf(-mt);
        sc[lane * 4 + 2] = expf(zf + before - mt);
        sc[lane * 4 + 3] = expf(zi - mt);
      }
      m = __shfl_sync(0xffffffffu, mt, n - 1);
    }
    __syncthreads();
    const ulonglong2* q = reinterpret_cast<const ulonglong2*>(sq) + l;
    const ulonglong2* k = reinterpret_cast<const ulonglong2*>(sk) + l;
    const ulonglong2* g = reinterpret_cast<const ulonglong2*>(sg) + l;
    const bool normaliser = KIND == kStateNormalized && c == a.vdim;
    const float* vc = sv + (c - c0);
    const bool vin = c < a.vdim;
    float* o = a.o + ((long long)r0 * a.heads + h) * a.vdim + c;
#pragma unroll 2
    for (int t = 0; t < n; ++t) {
      const float v = KIND == kStateNormalized && normaliser ? 1.f : vc[t * cols];
      float r = column_step<KIND, NV>(s, q + t * (DP / 4), k + t * (DP / 4), g + t * (DP / 4), v, sc[t * 4 + 2], sc[t * 4 + 3]);
      r = column_sum(r);
      if (KIND == kStateBonus) r = fmaf(sc[t * 4 + 2], v, r);
      if (l == 0) {
        if (vin) o[(long long)t * a.heads * a.vdim] = r * a.q_scale;
        else if (normaliser) *reinterpret_cast<float2*>(a.den + ((long long)(r0 + t) * a.heads + h) * 2) = make_float2(r * a.q_scale, sc[t * 4]);
      }
    }
    __syncthreads();                                                     // the stage is free again
  }

  if (live) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int e = (l + kLanes * i) * 4;
      if (e < d4) *reinterpret_cast<ulonglong2*>(now + at + e) = make_ulonglong2(s[2 * i], s[2 * i + 1]);
    }
  }
  if (KIND == kStateNormalized && blockIdx.x == 0 && threadIdx.x == 0) now[(long long)a.heads * C * d4 + h] = m;
  if (a.history) {
    const int keep = min(a.taps - 1, a.rows), ctas = gridDim.x * gridDim.y, cta = blockIdx.y * gridDim.x + blockIdx.x;
    for (int i = cta * blockDim.x + threadIdx.x; i < keep * a.hist_cols; i += ctas * blockDim.x) {
      const int j = a.rows - keep + i / a.hist_cols, cc = i % a.hist_cols;
      a.history[(long long)((pos0 + j) % a.hist_rows) * a.hist_cols + cc] = a.hist_src[(long long)j * a.hist_ld + cc];
    }
  }
  // A CTA that starts after this store still finds `pos0` in its own slot: only the other slot's tag changes.
  if (blockIdx.x == 0 && blockIdx.y == 0 && threadIdx.x == 0) {
    a.tags[1 - slot] = pos0 + a.rows;
    if (pos0 == 0) a.tags[1] = -1;
  }
}

// ------------------------------------------------------------------------------------ chunk path: around the recurrence
// One warp per (head or operand copy, strip of rows).
constexpr int kConvStrip = 8;

template <int NC>
__global__ void __launch_bounds__(128) short_conv_kernel(const ShortConvArgs a) {
  griddep_wait();
  griddep_launch();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seg = blockIdx.y * 4 + warp, r0 = blockIdx.x * kConvStrip, r1 = min(a.rows, r0 + kConvStrip);
  const int G = a.kv_heads, total = 2 * G + a.heads, columns = 2 * G * a.dim + a.heads * a.vdim;
  if (seg == total && a.low) {
    for (int r = r0; r < r1; ++r) {
      const float* p = a.proj + r * a.ld;
      for (int c = lane; c < a.low_cols; c += 32) store_act(a.low, r * a.low_ld + c, __ldg(p + a.low_off + c), a.f32);
      for (int c = lane; c < a.low2_cols; c += 32) store_act(a.low, r * a.low_ld + a.low2_at + c, __ldg(p + a.low2_off + c), a.f32);
    }
  }
  if (seg >= total) return;
  const int pos0 = *a.pos0;
  const bool is_v = seg >= 2 * G;
  const int w = is_v ? a.vdim : a.dim, col = is_v ? 2 * G * a.dim + (seg - 2 * G) * a.vdim : seg * a.dim;
  float* out = is_v ? a.v + (seg - 2 * G) * a.vdim : (seg < G ? a.q : a.k) + (seg % G) * a.dim;
  const long long out_ld = (long long)(is_v ? a.heads * a.vdim : G * a.dim);
  const __nv_bfloat16* kern = a.conv + (long long)col * a.taps;
  for (int r = r0; r < r1; ++r) {
    float y[NC], ss = 0.f;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = lane + 32 * i;
      y[i] = 0.f;
      if (c < w) {
#pragma unroll 4
        for (int j = 0; j < a.taps; ++j) {
          const int rr = r - (a.taps - 1 - j);
          float x = 0.f;
          if (rr >= 0) x = __ldg(a.proj + rr * a.ld + col + c);
          else if (pos0 + rr >= 0) x = a.history[(long long)((pos0 + rr) % a.hist_rows) * columns + col + c];
          y[i] = fmaf(bf(kern + c * a.taps + j), x, y[i]);
        }
        y[i] = silu_f(y[i]);
      }
      ss = fmaf(y[i], y[i], ss);
    }
    const float scale = is_v ? 1.f : (seg < G ? a.q_scale : 1.f) / sqrtf(lane_sum(ss) + kUnitEps);
#pragma unroll
    for (int i = 0; i < NC; ++i)
      if (lane + 32 * i < w) out[r * out_ld + lane + 32 * i] = y[i] * scale;
  }
}

__global__ void __launch_bounds__(256) token_mix_kernel(const TokenMixArgs a) {
  griddep_wait();
  griddep_launch();
  const int r = blockIdx.x, pos0 = *a.pos0;
  const int slot = state_slot(a.tags, pos0, a.status);
  if (slot < 0) return;
  const float* x = a.x + (long long)r * a.width;
  const float* before = r > 0 ? x - a.width : pos0 > 0 ? a.shift + slot * a.state_stride : nullptr;
  float* keep = r == a.rows - 1 ? a.shift + (1 - slot) * a.state_stride : nullptr;
  const long long o0 = (long long)r * a.mixes * a.out_ld;
  for (int c = threadIdx.x; c < a.width; c += 256) {
    const float v = __ldg(x + c), d = (before ? before[c] : 0.f) - v;
    for (int s = 0; s < a.mixes; ++s) store_act(a.out, o0 + s * a.out_ld + c, fmaf(d, bf(a.mu + (long long)s * a.width + c), v), a.f32);
    if (keep) keep[c] = v;
  }
}

// One warp per (row, head).
__global__ void __launch_bounds__(256) head_gate_kernel(const HeadGateArgs a) {
  griddep_wait();
  griddep_launch();
  const int lane = threadIdx.x & 31, r = blockIdx.x, h = blockIdx.y * 8 + (threadIdx.x >> 5);
  if (h >= a.heads) return;
  const float* o = a.o + ((long long)r * a.heads + h) * a.vdim;
  float inv = 1.f;
  if (a.den) {
    const float* d = a.den + ((long long)r * a.heads + h) * 2;
    inv = 1.0f / (fmaxf(fabsf(d[0]), d[1]) + 1e-6f);
  }
  float ss = 0.f;
  for (int c = lane; c < a.vdim; c += 32) {
    const float v = __ldg(o + c) * inv;
    ss = fmaf(v, v, ss);
  }
  const float rs = inv / sqrtf(lane_sum(ss) / (float)a.vdim + a.eps);
  const float* g = a.gate + (long long)r * a.gate_ld + (long long)h * a.vdim;
  const __nv_bfloat16* w = a.norm + (a.norm_per_head ? (long long)h * a.vdim : 0);
  for (int c = lane; c < a.vdim; c += 32) {
    const float z = __ldg(g + c), gate = a.gate_kind == kGateSilu ? silu_f(z) : sigmoid_f(z);
    store_act(a.out, (long long)r * a.out_ld + (long long)h * a.vdim + c, __ldg(o + c) * rs * bf(w + c) * gate, a.f32);
  }
}

// ------------------------------------------------------------------------------------ one token
// One CTA per head.  The state is requested before the wait for the predecessor: it was written a whole step ago.
constexpr int kStepT = 512, kStepCols = kStepT / kLanes;

// rows of a low-rank product: out[row] = W[row] . in, one warp per row
template <class F>
__device__ __forceinline__ void low_rank_rows(const __nv_bfloat16* w, long long ld, int rows, const float* in, int warp, int lane, F store) {
#pragma unroll 4
  for (int r = warp; r < rows; r += kStepT / 32) {
    float acc = 0.f;
    for (int c = lane * 4; c < (int)ld; c += 128) {
      const uint2 p = __ldg(reinterpret_cast<const uint2*>(w + r * ld + c));
      const float4 x = *reinterpret_cast<const float4*>(in + c);
      acc = fmaf(bf16_lo(p.x), x.x, fmaf(bf16_hi(p.x), x.y, fmaf(bf16_lo(p.y), x.z, fmaf(bf16_hi(p.y), x.w, acc))));
    }
    acc = lane_sum(acc);
    if (lane == 0) store(r, acc);
  }
}
__host__ __device__ inline int step_floats(int dp, int vdim, int decay_ld, int gate_ld) {
  return 3 * dp + 2 * pad4(vdim + 1) + decay_ld + gate_ld;
}

template <int KIND, int NV>
__global__ void __launch_bounds__(kStepT) state_step_kernel(const StateStepArgs a) {
  constexpr int DP = NV * 4 * kLanes, AHEAD = NV <= 4 ? 2 : 1;
  extern __shared__ __align__(16) float sh[];
  __shared__ float red[33];
  float* sk = sh;
  float* sq = sk + DP;
  float* sg = sq + DP;
  float* so = sg + DP;
  float* sgate = so + pad4(a.vdim + 1);
  float* slow = sgate + pad4(a.vdim + 1);
  float* sgin = slow + a.decay_ld;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, l = lane & (kLanes - 1);
  const int C = a.vdim + extra_columns<KIND>(), d4 = pad4(a.dim), h = blockIdx.x, hk = h / (a.heads / a.kv_heads);
  const int pos = *reinterpret_cast<const volatile int*>(a.pos0);
  const int slot = state_slot(a.tags, pos, a.status);
  const float* old = a.state + max(slot, 0) * a.state_stride + (long long)h * C * d4;
  float* now = a.state + (1 - max(slot, 0)) * a.state_stride + (long long)h * C * d4;
  auto load = [&](int c, u64 (&s)[2 * NV]) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int e = (l + kLanes * i) * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < C && pos > 0 && e < d4) v = __ldcg(reinterpret_cast<const float4*>(old + (long long)c * d4 + e));
      s[2 * i] = pack2(v.x, v.y);
      s[2 * i + 1] = pack2(v.z, v.w);
    }
  };
  u64 first[AHEAD][2 * NV];
#pragma unroll
  for (int j = 0; j < AHEAD; ++j) load(threadIdx.x / kLanes + j * kStepCols, first[j]);
  griddep_wait();
  griddep_launch();
  if (slot < 0) return;
  const float* p = a.proj;
  for (int i = threadIdx.x; i < DP; i += kStepT) {
    const bool in = i < a.dim;
    sk[i] = in ? __ldcg(p + a.k_off + hk * a.dim + i) : 0.f;
    sq[i] = in ? __ldcg(p + a.q_off + hk * a.dim + i) : 0.f;
    sg[i] = 0.f;
  }
  if (KIND != kStateNormalized)
    for (int i = threadIdx.x; i < a.decay_ld; i += kStepT) {
      const float z = i < a.low_rank ? __ldcg(p + a.low_off + i) : 0.f;
      slow[i] = a.low_tanh ? tanhf(z) : z;
    }
  if (a.gate_w)
    for (int i = threadIdx.x; i < a.gate_ld; i += kStepT) sgin[i] = i < a.gate_rank ? __ldcg(p + a.gate_off + i) : 0.f;
  __syncthreads();
  if (KIND != kStateNormalized) {
    const __nv_bfloat16* b = a.decay_b + (long long)h * a.dim;
    const float* rate = a.rate ? a.rate + (long long)h * a.dim : nullptr;
    low_rank_rows(a.decay_w + (long long)h * a.dim * a.decay_ld, a.decay_ld, a.dim, slow, warp, lane, [&](int d, float z) {
      z += bf(b + d);
      sg[d] = rate ? decay_soft(z, rate[d]) : decay_exp(z);
    });
  }
  if (a.gate_w)
    low_rank_rows(a.gate_w + (long long)h * a.vdim * a.gate_ld, a.gate_ld, a.vdim, sgin, warp, lane, [&](int j, float z) { sgate[j] = z; });
  else
    for (int j = threadIdx.x; j < a.vdim; j += kStepT) sgate[j] = __ldcg(p + a.gate_off + (long long)h * a.vdim + j);
  float q_scale = a.q_scale;
  if (a.unit) {
    float qq = 0.f, kk = 0.f;
    for (int i = lane; i < a.dim; i += 32) {
      qq = fmaf(sq[i], sq[i], qq);
      kk = fmaf(sk[i], sk[i], kk);
    }
    q_scale /= sqrtf(lane_sum(qq) + kUnitEps);
    const float ks = 1.0f / sqrtf(lane_sum(kk) + kUnitEps);
    __syncthreads();
    for (int i = threadIdx.x; i < a.dim; i += kStepT) sk[i] *= ks;
  }
  float s0 = 0.f, s1 = 0.f, floor_n = 0.f, m_new = 0.f;
  if (KIND == kStateDelta) s0 = sigmoid_f(__ldcg(p + a.beta_off + h));
  if (KIND == kStateNormalized) {
    const float zi = log_input(__ldcg(p + a.gi_off + h), a.cap), zf = log_forget(__ldcg(p + a.gf_off + h), a.cap);
    const long long m_at = (long long)(a.heads - h) * C * d4 + h;        // the maxima follow the last head's state
    const float m = pos > 0 ? __ldcg(old + m_at) : 0.f;
    m_new = fmaxf(zf + m, zi);
    s0 = expf(zf + m - m_new);
    s1 = expf(zi - m_new);
    floor_n = expf(-m_new);
    if (threadIdx.x == 0) now[m_at] = m_new;
  }
  if (KIND == kStateBonus) {
    for (int i = lane; i < a.dim; i += 32) s0 = fmaf(sq[i] * bf(a.u + (long long)h * a.dim + i), sk[i], s0);
    s0 = lane_sum(s0);
  }
  __syncthreads();
  const ulonglong2* q = reinterpret_cast<const ulonglong2*>(sq) + l;
  const ulonglong2* k = reinterpret_cast<const ulonglong2*>(sk) + l;
  const ulonglong2* g = reinterpret_cast<const ulonglong2*>(sg) + l;
  auto column = [&](int c, u64 (&s)[2 * NV]) {
    const float v = c < a.vdim ? __ldcg(p + a.v_off + (long long)h * a.vdim + c) : c < C ? 1.f : 0.f;
    float r = column_sum(column_step<KIND, NV>(s, q, k, g, v, s0, s1));
    if (KIND == kStateBonus) r = fmaf(s0, v, r);
    if (c < C) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int e = (l + kLanes * i) * 4;
        if (e < d4) *reinterpret_cast<ulonglong2*>(now + (long long)c * d4 + e) = make_ulonglong2(s[2 * i], s[2 * i + 1]);
      }
      if (l == 0) so[c] = r * q_scale;
    }
  };
#pragma unroll
  for (int j = 0; j < AHEAD; ++j) column(threadIdx.x / kLanes + j * kStepCols, first[j]);
  for (int cb = AHEAD * kStepCols; cb < C; cb += kStepCols) {            // (the same trip count for every lane of a warp)
    u64 s[2 * NV];
    load(cb + threadIdx.x / kLanes, s);
    column(cb + threadIdx.x / kLanes, s);
  }
  __syncthreads();
  const float inv = KIND == kStateNormalized ? 1.0f / (fmaxf(fabsf(so[a.vdim]), floor_n) + 1e-6f) : 1.f;
  float ss = 0.f;
  for (int j = threadIdx.x; j < a.vdim; j += kStepT) {
    const float v = so[j] * inv;
    ss = fmaf(v, v, ss);
  }
  const float rs = inv / sqrtf(block_sum_f(ss, red) / (float)a.vdim + a.eps);
  const __nv_bfloat16* w = a.norm + (a.norm_per_head ? (long long)h * a.vdim : 0);
  for (int j = threadIdx.x; j < a.vdim; j += kStepT)
    a.out[(long long)h * a.vdim + j] = so[j] * rs * bf(w + j) * (a.gate_kind == kGateSilu ? silu_f(sgate[j]) : sigmoid_f(sgate[j]));
  // A CTA that starts after this store still finds `pos` in its own slot: only the other slot's tag changes.
  if (blockIdx.x == 0 && threadIdx.x == 0) {
    a.tags[1 - slot] = pos + 1;
    if (pos == 0) a.tags[1] = -1;
  }
}

constexpr int kMaxSmem = 220 * 1024;

template <class K>
int allow_smem(K kern, bool& done) {
  if (done) return 0;
  const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxSmem);
  done = e == cudaSuccess;
  return (int)e;
}

template <int KIND, int NV>
int launch_chunk(const StateChunkArgs& a, cudaStream_t stream) {
  static bool configured = false;
  if (const int rc = allow_smem(state_chunk_kernel<KIND, NV>, configured)) return rc;
  const int C = a.vdim + extra_columns<KIND>();
  int warps = 8;
  while (warps > 2 && a.heads * ((C + warps * 4 - 1) / (warps * 4)) < 100) warps /= 2;
  const int cols = warps * 4;
  int tokens = 32;
  while (tokens > 4 && 8 * chunk_stage_floats(KIND, NV * 4 * kLanes, cols, tokens) > 110 * 1024) tokens /= 2;
  const int smem = 8 * chunk_stage_floats(KIND, NV * 4 * kLanes, cols, tokens);
  return launch_pdl(state_chunk_kernel<KIND, NV>, dim3((C + cols - 1) / cols, a.heads), dim3(warps * 32), smem, stream, false, a, tokens);
}
template <int KIND, int NV>
int launch_state_step(const StateStepArgs& a, cudaStream_t stream, bool pdl) {
  static bool configured = false;
  if (const int rc = allow_smem(state_step_kernel<KIND, NV>, configured)) return rc;
  const int smem = 4 * step_floats(NV * 4 * kLanes, a.vdim, (int)a.decay_ld, (int)a.gate_ld);
  if (smem > kMaxSmem) return -7;
  return launch_pdl(state_step_kernel<KIND, NV>, dim3(a.heads), dim3(kStepT), smem, stream, pdl, a);
}

bool sizes_ok(int heads, int kv_heads, int dim, int vdim) {
  return heads >= 1 && kv_heads >= 1 && heads % kv_heads == 0 && dim >= 1 && dim <= 512 && vdim >= 1;
}

}  // namespace

#define S(stream) reinterpret_cast<cudaStream_t>(stream)
// pieces of 16 bytes per lane and column
#define NRT_BY_DIM(CALL, KIND, dim, ...)                       \
  if ((dim) <= 32) return CALL<KIND, 1>(__VA_ARGS__);          \
  if ((dim) <= 64) return CALL<KIND, 2>(__VA_ARGS__);          \
  if ((dim) <= 128) return CALL<KIND, 4>(__VA_ARGS__);         \
  if ((dim) <= 256) return CALL<KIND, 8>(__VA_ARGS__);         \
  return CALL<KIND, 16>(__VA_ARGS__);

extern "C" int nrt_state_chunk_args_size() { return (int)sizeof(StateChunkArgs); }
extern "C" int nrt_short_conv_args_size() { return (int)sizeof(ShortConvArgs); }
extern "C" int nrt_token_mix_args_size() { return (int)sizeof(TokenMixArgs); }
extern "C" int nrt_head_gate_args_size() { return (int)sizeof(HeadGateArgs); }
extern "C" int nrt_state_step_args_size() { return (int)sizeof(StateStepArgs); }

extern "C" int nrt_state_chunk(int kind, const void* args, void* stream) {
  StateChunkArgs a;
  memcpy(&a, args, sizeof(a));
  if (a.rows < 1 || !sizes_ok(a.heads, a.kv_heads, a.dim, a.vdim) || a.state_stride % 4) return -3;
  if (a.history && (a.hist_rows < 1 || a.hist_rows < 2 * (a.taps - 1))) return -3;
  if ((kind != kStateNormalized && !a.g) || (kind == kStateNormalized && (!a.gi || !a.gf || !a.den)) || (kind == kStateDelta && !a.beta) || (kind == kStateBonus && !a.u)) return -3;
  if (kind == kStateDelta) { NRT_BY_DIM(launch_chunk, kStateDelta, a.dim, a, S(stream)) }
  if (kind == kStateBonus) { NRT_BY_DIM(launch_chunk, kStateBonus, a.dim, a, S(stream)) }
  if (kind == kStateNormalized) { NRT_BY_DIM(launch_chunk, kStateNormalized, a.dim, a, S(stream)) }
  return -2;
}

extern "C" int nrt_state_step(const void* args, void* stream, int pdl) {
  StateStepArgs a;
  memcpy(&a, args, sizeof(a));
  if (!sizes_ok(a.heads, a.kv_heads, a.dim, a.vdim) || a.state_stride % 4 || a.decay_ld % 8 || a.gate_ld % 8 || !a.norm) return -3;
  if ((kStateNormalized != a.kind && (!a.decay_w || !a.decay_b || a.low_rank > a.decay_ld)) || (a.gate_w && a.gate_rank > a.gate_ld)) return -3;
  if (a.kind == kStateBonus && !a.u) return -3;
  const bool p = pdl != 0;
  if (a.kind == kStateDelta) { NRT_BY_DIM(launch_state_step, kStateDelta, a.dim, a, S(stream), p) }
  if (a.kind == kStateBonus) { NRT_BY_DIM(launch_state_step, kStateBonus, a.dim, a, S(stream), p) }
  if (a.kind == kStateNormalized) { NRT_BY_DIM(launch_state_step, kStateNormalized, a.dim, a, S(stream), p) }
  return -2;
}

extern "C" int nrt_short_conv(const void* args, void* stream) {
  ShortConvArgs a;
  memcpy(&a, args, sizeof(a));
  if (a.rows < 1 || a.taps < 1 || !sizes_ok(a.heads, a.kv_heads, a.dim, a.vdim) || a.vdim > 512 || a.hist_rows < 1 || a.hist_rows < 2 * (a.taps - 1)) return -3;
  const dim3 grid((a.rows + kConvStrip - 1) / kConvStrip, (2 * a.kv_heads + a.heads + 1 + 3) / 4);
  const int w = a.dim > a.vdim ? a.dim : a.vdim;
  if (w <= 32) return launch_pdl(short_conv_kernel<1>, grid, dim3(128), 0, S(stream), false, a);
  if (w <= 64) return launch_pdl(short_conv_kernel<2>, grid, dim3(128), 0, S(stream), false, a);
  if (w <= 128) return launch_pdl(short_conv_kernel<4>, grid, dim3(128), 0, S(stream), false, a);
  if (w <= 256) return launch_pdl(short_conv_kernel<8>, grid, dim3(128), 0, S(stream), false, a);
  return launch_pdl(short_conv_kernel<16>, grid, dim3(128), 0, S(stream), false, a);
}

extern "C" int nrt_token_mix(const void* args, void* stream) {
  TokenMixArgs a;
  memcpy(&a, args, sizeof(a));
  if (a.rows < 1 || a.width < 1 || a.mixes < 1) return -3;
  return launch_pdl(token_mix_kernel, dim3(a.rows), dim3(256), 0, S(stream), false, a);
}

extern "C" int nrt_head_gate(const void* args, void* stream) {
  HeadGateArgs a;
  memcpy(&a, args, sizeof(a));
  if (a.rows < 1 || a.heads < 1 || a.vdim < 1 || !a.gate || !a.norm) return -3;
  return launch_pdl(head_gate_kernel, dim3(a.rows, (a.heads + 7) / 8), dim3(256), 0, S(stream), false, a);
}
