// One-token step of layer stacks: matrix-vector products with their surroundings fused in.
//
// A single token reads every weight once, so the step is bound by HBM and the CUDA cores keep up with it; activations stay
// fp32 throughout.  Each launch is (prologue) -> W h -> (epilogue):
//   prologues  stream update + norm (every CTA repeats it: two row-sized L2 reads instead of a launch of its own), norm of a
//              segment, plain load per group, merge of the attention partials
//   epilogues  store / sigmoid, biased branches with the short convolution, output gate, two-product activations, the
//              recurrence step
// The first weights of a CTA are requested before griddepcontrol.wait: with programmatic dependent launch they travel under
// the predecessor's tail.
#include "stack.cuh"
#include "launch.hpp"
#include "router.cuh"

#include <string.h>

using namespace nrt;

namespace {

constexpr int kStepThreads = 256;

// The input vector lives in shared memory as two planes of float4: chunk c of eight elements is plane0[c], plane1[c], so that
// neighbouring lanes read neighbouring 16-byte words.
__device__ __forceinline__ int plane_at(int c, int k8) { return ((c >> 2) & 1) * k8 * 4 + (c >> 3) * 4 + (c & 3); }

__device__ __forceinline__ float dot8(const uint4& w, const float4& a, const float4& b, float acc) {
  acc = fmaf(bf16_lo(w.x), a.x, acc);
  acc = fmaf(bf16_hi(w.x), a.y, acc);
  acc = fmaf(bf16_lo(w.y), a.z, acc);
  acc = fmaf(bf16_hi(w.y), a.w, acc);
  acc = fmaf(bf16_lo(w.z), b.x, acc);
  acc = fmaf(bf16_hi(w.z), b.y, acc);
  acc = fmaf(bf16_lo(w.w), b.z, acc);
  acc = fmaf(bf16_hi(w.w), b.w, acc);
  return acc;
}
__device__ __forceinline__ uint4 ld_stream(const uint4* p) {           // weights: read once per step
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.b32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}

// Values of the first kPreSpan elements that do not depend on the predecessor kernel, requested before the wait for it: the
// norm weights, and the stream itself (written at least two launches back).
constexpr int kPreSpan = kStepThreads * 16;
struct Pre {
  float4 x[4];
  uint2 post[4], in[4];
};
__device__ __forceinline__ float4 bf4(const uint2& v) { return make_float4(bf16_lo(v.x), bf16_hi(v.x), bf16_lo(v.y), bf16_hi(v.y)); }
__device__ __forceinline__ float4 ldcg4(const float* p) { return __ldcg(reinterpret_cast<const float4*>(p)); }
__device__ __forceinline__ uint2 ldw4(const __nv_bfloat16* p) { return __ldg(reinterpret_cast<const uint2*>(p)); }
__device__ __forceinline__ float dot4(const float4& v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
__device__ __forceinline__ float4 fma4(const float4& a, const float4& b, float s, const float4& c) {      // a * b * s + c
  return make_float4(fmaf(a.x * s, b.x, c.x), fmaf(a.y * s, b.y, c.y), fmaf(a.z * s, b.z, c.z), fmaf(a.w * s, b.w, c.w));
}

template <int PRO>
__device__ __forceinline__ void preload(const StepArgs& a, Pre& p) {
  if (a.k & 3) return;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int e = (i * kStepThreads + (int)threadIdx.x) * 4;
    p.x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    p.post[i] = p.in[i] = make_uint2(0u, 0u);
    if (e < a.k) {
      p.in[i] = ldw4(a.in_w + e);
      if (PRO == kProResidual) {
        if (a.y) p.post[i] = ldw4(a.post_w + e);
        if (!a.tokens) p.x[i] = ldcg4(a.x + e);
      }
    }
  }
}

template <int PRO>
__device__ __forceinline__ void load_input(const StepArgs& a, int g, int k8, float* hs, float* red, const Pre& p, int pos) {
  const int K = a.k;
  float4* hs4 = reinterpret_cast<float4*>(hs);
  // element e (a multiple of four) of the input -> its float4 in the two planes
  auto at4 = [&](int e) -> float4& { return hs4[((e >> 2) & 1) * k8 + (e >> 3)]; };
  if (PRO == kProResidual || PRO == kProNorm) {
    const __nv_bfloat16* emb = nullptr;
    if (PRO == kProResidual && a.tokens) {
      int t = *reinterpret_cast<const volatile int*>(a.tokens);
      t = t < 0 ? 0 : t >= a.vocab ? a.vocab - 1 : t;
      emb = a.table + (size_t)t * K;
    }
    if ((K & 3) == 0) {
      float4 v[4];
      float ss = 0.f, sq = 0.f;
      if (PRO == kProResidual && a.y) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int e = (i * kStepThreads + (int)threadIdx.x) * 4;
          v[i] = e < K ? ldcg4(a.y + e) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) ss += dot4(v[i]);
        for (int e = kPreSpan + (int)threadIdx.x * 4; e < K; e += kStepThreads * 4) ss += dot4(ldcg4(a.y + e));
        ss = block_sum_f(ss, red);
      } else if (PRO == kProNorm) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int e = (i * kStepThreads + (int)threadIdx.x) * 4;
          v[i] = e < K ? ldcg4(a.in_ + e) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
      }
      const float ry = PRO == kProResidual && a.y ? 1.0f / sqrtf(ss / (float)K + a.eps) : 0.f;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int e = (i * kStepThreads + (int)threadIdx.x) * 4;
        if (e >= K) continue;
        if (PRO == kProResidual) {
          float4 x = p.x[i];
          if (emb) { const float4 t = bf4(ldw4(emb + e)); x = make_float4(t.x * a.embed_scale, t.y * a.embed_scale, t.z * a.embed_scale, t.w * a.embed_scale); }
          if (a.y) x = fma4(v[i], bf4(p.post[i]), ry, x);
          if (a.add) { const float4 t = bf4(ldw4(a.add + e)); x = make_float4(x.x + t.x, x.y + t.y, x.z + t.z, x.w + t.w); }
          if (blockIdx.x == 0) *reinterpret_cast<float4*>(a.x_out + e) = x;
          v[i] = x;
        }
        sq += dot4(v[i]);
      }
      for (int e = kPreSpan + (int)threadIdx.x * 4; e < K; e += kStepThreads * 4) {
        float4 x;
        if (PRO == kProResidual) {
          if (emb) { const float4 t = bf4(ldw4(emb + e)); x = make_float4(t.x * a.embed_scale, t.y * a.embed_scale, t.z * a.embed_scale, t.w * a.embed_scale); }
          else x = ldcg4(a.x + e);
          if (a.y) x = fma4(ldcg4(a.y + e), bf4(ldw4(a.post_w + e)), ry, x);
          if (a.add) { const float4 t = bf4(ldw4(a.add + e)); x = make_float4(x.x + t.x, x.y + t.y, x.z + t.z, x.w + t.w); }
          if (blockIdx.x == 0) *reinterpret_cast<float4*>(a.x_out + e) = x;
        } else {
          x = ldcg4(a.in_ + e);
        }
        at4(e) = x;
        sq += dot4(x);
      }
      sq = block_sum_f(sq, red);
      const float rx = 1.0f / sqrtf(sq / (float)K + a.eps);
      const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int e = (i * kStepThreads + (int)threadIdx.x) * 4;
        if (e < K) at4(e) = fma4(v[i], bf4(p.in[i]), rx, zero);
      }
      for (int e = kPreSpan + (int)threadIdx.x * 4; e < K; e += kStepThreads * 4) at4(e) = fma4(at4(e), bf4(ldw4(a.in_w + e)), rx, zero);
    } else {
      float ss = 0.f, sq = 0.f;
      if (PRO == kProResidual && a.y) {
        for (int c = threadIdx.x; c < K; c += kStepThreads) { const float v = __ldcg(a.y + c); ss = fmaf(v, v, ss); }
        ss = block_sum_f(ss, red);
      }
      const float ry = PRO == kProResidual && a.y ? 1.0f / sqrtf(ss / (float)K + a.eps) : 0.f;
      for (int c = threadIdx.x; c < K; c += kStepThreads) {
        float v = PRO == kProNorm ? __ldcg(a.in_ + c) : emb ? bf(emb + c) * a.embed_scale : __ldcg(a.x + c);
        if (PRO == kProResidual) {
          if (a.y) v += __ldcg(a.y + c) * ry * bf(a.post_w + c);
          if (a.add) v += bf(a.add + c);
          if (blockIdx.x == 0) a.x_out[c] = v;
        }
        hs[plane_at(c, k8)] = v;
        sq = fmaf(v, v, sq);
      }
      sq = block_sum_f(sq, red);
      const float rx = 1.0f / sqrtf(sq / (float)K + a.eps);
      for (int c = threadIdx.x; c < K; c += kStepThreads) hs[plane_at(c, k8)] *= rx * bf(a.in_w + c);
    }
  } else if (PRO == kProLoad) {
    const float* in = a.in_ + g * a.in_gstride;
    if (((K | (int)a.in_gstride) & 3) == 0) {
#pragma unroll 4
      for (int e = (int)threadIdx.x * 4; e < K; e += kStepThreads * 4) at4(e) = ldcg4(in + e);
    } else {
      for (int c = threadIdx.x; c < K; c += kStepThreads) hs[plane_at(c, k8)] = __ldcg(in + c);
    }
  } else {                                                             // kProMerge
    // weights of the used splits, then a weighted sum of their outputs; threads beyond the row's float4 columns take other splits
    __shared__ float ws[kMaxSplits];
    const int n = pos + 1, per = latent_split_rows(n, a.splits), used = (n + per - 1) / per;
    const int row = latent_part_row(K), k4 = (K + 3) / 4;
    const size_t hstride = (size_t)a.groups * row;
    const float* p0 = a.part + (size_t)g * row;
    float ms = -FLT_MAX, ls = 0.f;
    if ((int)threadIdx.x < used) { ms = __ldcg(p0 + threadIdx.x * hstride); ls = __ldcg(p0 + threadIdx.x * hstride + 1); }
    float m = ms;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = m;
    __syncthreads();
#pragma unroll
    for (int i = 0; i < kStepThreads / 32; ++i) m = fmaxf(m, red[i]);
    const float w = (int)threadIdx.x < used ? expf(ms - m) : 0.f;
    const float l = block_sum_f(ls * w, red);
    if ((int)threadIdx.x < used) ws[threadIdx.x] = w / l;
    int cols = 1;
    while (cols < k4 && cols < kStepThreads) cols *= 2;
    const int subs = kStepThreads / cols, sub = (int)threadIdx.x / cols, c0 = (int)threadIdx.x & (cols - 1);
    __syncthreads();
    for (int i = threadIdx.x; i < 2 * k8; i += kStepThreads) hs4[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    __syncthreads();
    for (int cb = 0; cb < k4; cb += cols) {
      const int c = cb + c0;
      float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
      for (int s = sub; s < used && c < k4; s += subs) {
        const float4 v = ldcg4(p0 + s * hstride + 4 + c * 4);
        const float wv = ws[s];
        acc = make_float4(fmaf(v.x, wv, acc.x), fmaf(v.y, wv, acc.y), fmaf(v.z, wv, acc.z), fmaf(v.w, wv, acc.w));
      }
      // sub-sums join in a fixed order
      for (int q = 0; q < subs; ++q) {
        if (sub == q && c < k4) { float4& d = at4(c * 4); d = make_float4(d.x + acc.x, d.y + acc.y, d.z + acc.z, d.w + acc.w); }
        if (subs > 1) __syncthreads();
      }
    }
    __syncthreads();
  }
  for (int c = K + threadIdx.x; c < k8 * 8; c += kStepThreads) hs[plane_at(c, k8)] = 0.f;
  __syncthreads();
}

template <int EPI>
__device__ __forceinline__ void finish_row(const StepArgs& a, int g, int row, float v, float v2, int pos, int slot) {
  const size_t at = (size_t)g * a.n + row;
  if (EPI == kTEpiStore) {
    a.out[at] = row >= a.sig_from ? sigmoid_f(v) : v * a.scale;
  } else if (EPI == kTEpiGate) {
    a.out[at] = v * __ldcg(a.gate + at);
  } else if (EPI == kTEpiGlu) {
    a.out[at] = a.glu_kind == 0 ? clamped_glu(v, v2, a.limit, a.alpha) : silu_glu(v, v2);
  } else if (EPI == kTEpiConv) {
    const int width = a.n / 2;
    v += bf(a.bias + row);
    if (row < width) {
      v = gelu_tanh_f(v);
      a.out[row] = a.f32 ? v : round_bf16(v);
    } else {
      const int c = row - width;
      const float x = a.f32 ? v : round_bf16(v);
      float u = bf(a.conv_b + c);
      for (int j = 0; j < a.taps - 1; ++j) {
        const int back = a.taps - 1 - j;
        if (back <= pos) u = fmaf(bf(a.conv + (size_t)c * a.taps + j), a.history[(long long)((pos - back) % a.hist_rows) * width + c], u);
      }
      u = fmaf(bf(a.conv + (size_t)c * a.taps + a.taps - 1), x, u);
      a.u[c] = a.f32 ? u : round_bf16(u);
      a.history[(long long)(pos % a.hist_rows) * width + c] = x;
    }
  } else {                                                             // kTEpiRecur
    const int c = (int)at, width = a.groups * a.n;
    const float rg = sigmoid_f(v + bf(a.bias + c)), ig = sigmoid_f(v2 + bf(a.bias2 + c));
    const float la = -a.decay * rg * a.softplus_lam[c];
    const float prev = pos == 0 ? 0.f : a.state[(size_t)slot * width + c];
    const float s = fmaf(expf(la), prev, sqrtf(-expm1f(2.0f * la)) * ig * __ldcg(a.u + c));
    a.state[(size_t)(1 - slot) * width + c] = s;
    a.out[c] = s * __ldcg(a.gate + c);
  }
}

constexpr int kMaxStepSmem = 200 * 1024;

template <int PRO, int EPI, int RU, int U, bool ROUTE>
__global__ void __launch_bounds__(kStepThreads) stack_step_kernel(const StepArgs a, const RouterArgs ra, const int rgroups,
                                                                  const int rkeep, const int G) {
  constexpr bool DUAL = EPI == kTEpiGlu || EPI == kTEpiRecur;
  constexpr bool PER_GROUP = PRO == kProLoad || PRO == kProMerge;
  extern __shared__ float4 hs4[];
  __shared__ float red[33];
  __shared__ int s_ids[32];
  float* hs = reinterpret_cast<float*>(hs4);
  const int k8 = (a.k + 7) / 8;
  const int lig = threadIdx.x & (G - 1), grp = threadIdx.x / G, gpc = kStepThreads / G;
  const int rows_tile = gpc * RU;
  const int tiles_g = (a.n + rows_tile - 1) / rows_tile;
  const int tiles = a.groups * tiles_g;
  uint4 wv[RU][U], wv2[DUAL ? RU : 1][DUAL ? U : 1];

  auto fetch = [&](int tile, int c0) {
    const int g = tile / tiles_g;
    const int wg = ROUTE ? s_ids[g] : g;
    const int row0 = (tile - g * tiles_g) * rows_tile + grp * RU;
#pragma unroll
    for (int i = 0; i < RU; ++i) {
      const bool in = row0 + i < a.n;
      const uint4* p = reinterpret_cast<const uint4*>(a.w + wg * a.w_gstride + (long long)(row0 + i) * a.w_ld);
      const uint4* p2 = DUAL ? reinterpret_cast<const uint4*>(a.w2 + wg * a.w2_gstride + (long long)(row0 + i) * a.w_ld) : nullptr;
#pragma unroll
      for (int q = 0; q < U; ++q) {
        const int c = c0 + q * G;
        wv[i][q] = in && c < k8 ? ld_stream(p + c) : make_uint4(0u, 0u, 0u, 0u);
        if (DUAL) wv2[DUAL ? i : 0][DUAL ? q : 0] = in && c < k8 ? ld_stream(p2 + c) : make_uint4(0u, 0u, 0u, 0u);
      }
    }
  };

  // each CTA owns a contiguous run of tiles, so a per-group input is loaded once per group it meets
  const int per_cta = (tiles + (int)gridDim.x - 1) / (int)gridDim.x;
  const int tile_lo = (int)blockIdx.x * per_cta, tile_hi = min(tiles, tile_lo + per_cta);
  if (!ROUTE && tile_lo < tile_hi) fetch(tile_lo, lig);
  Pre pre;
  if constexpr (PRO == kProResidual) preload<PRO>(a, pre);       // (a normed input vector may come from the predecessor itself)
  griddep_wait();
  griddep_launch();
  const int pos = a.pos0 ? *reinterpret_cast<const volatile int*>(a.pos0) : 0;
  if (ROUTE) {
    __shared__ RouterSmem sm;
    router_select<true>(ra, sm, blockIdx.x == 0, nullptr, nullptr, nullptr, rgroups, rkeep);
    __syncthreads();
    if ((int)threadIdx.x < ra.top_k) s_ids[threadIdx.x] = sm.tk_id[0][threadIdx.x];
    __syncthreads();
  }
  int slot = 1;
  if (EPI == kTEpiRecur) {
    slot = state_slot(a.tags, pos, a.status);
    if (slot < 0) return;
  }
  if constexpr (PRO == kProNorm) preload<PRO>(a, pre);
  if (!PER_GROUP) load_input<PRO>(a, 0, k8, hs, red, pre, pos);
  if (PRO == kProNorm && a.lat_in && blockIdx.x == gridDim.x - 1 && pos >= 0 && pos < a.capacity) {
    // append the token's key/value latent to the cache
    float sq = 0.f;
    for (int c = threadIdx.x; c < a.lat_rank; c += kStepThreads) { const float v = __ldcg(a.lat_in + c); sq = fmaf(v, v, sq); }
    const float rs = 1.0f / sqrtf(block_sum_f(sq, red) / (float)a.lat_rank + a.eps);
    for (int c = threadIdx.x; c < a.lat_rank; c += kStepThreads)
      store_act(a.lat_cache, (long long)pos * a.lat_ld + c, __ldcg(a.lat_in + c) * rs * bf(a.lat_w + c), a.f32);
  }
  int cur = -1;
  for (int tile = tile_lo; tile < tile_hi; ++tile) {
    const int g = tile / tiles_g;
    if (PER_GROUP && g != cur) {
      if (cur >= 0) __syncthreads();
      load_input<PRO>(a, g, k8, hs, red, pre, pos);
      cur = g;
    }
    float acc[RU], acc2[RU];
#pragma unroll
    for (int i = 0; i < RU; ++i) acc[i] = acc2[i] = 0.f;
#pragma unroll 1
    for (int c0 = lig; c0 < k8 || c0 == lig; c0 += G * U) {
      if (c0 != lig || ROUTE || tile != tile_lo) fetch(tile, c0);
#pragma unroll
      for (int q = 0; q < U; ++q) {
        const int c = c0 + q * G;
        if (c < k8) {
          const float4 x0 = hs4[c], x1 = hs4[k8 + c];
#pragma unroll
          for (int i = 0; i < RU; ++i) {
            acc[i] = dot8(wv[i][q], x0, x1, acc[i]);
            if (DUAL) acc2[i] = dot8(wv2[DUAL ? i : 0][DUAL ? q : 0], x0, x1, acc2[i]);
          }
        }
      }
    }
#pragma unroll
    for (int i = 0; i < RU; ++i)
      for (int o = G >> 1; o > 0; o >>= 1) {
        acc[i] += __shfl_xor_sync(0xffffffffu, acc[i], o);
        if (DUAL) acc2[i] += __shfl_xor_sync(0xffffffffu, acc2[i], o);
      }
    if (lig == 0) {
      const int row0 = (tile - g * tiles_g) * rows_tile + grp * RU;
#pragma unroll
      for (int i = 0; i < RU; ++i)
        if (row0 + i < a.n) finish_row<EPI>(a, g, row0 + i, acc[i], acc2[i], pos, slot);
    }
    __syncwarp();
  }
  // A CTA that starts after this store still finds `pos` in its own slot: only the other slot's tag changes.
  if (EPI == kTEpiRecur && blockIdx.x == 0 && threadIdx.x == 0) {
    a.tags[1 - slot] = pos + 1;
    if (pos == 0) a.tags[1] = -1;
  }
}

// Second product of the routed experts: out[n] = sum_j p_j (W[id_j] act_j)[n], warp per RU rows.
template <int RU, int U>
__global__ void __launch_bounds__(kStepThreads) stack_down_kernel(const StepDownArgs a) {
  extern __shared__ float4 hs4[];
  __shared__ int s_ids[32];
  float* hs = reinterpret_cast<float*>(hs4);
  const int k8 = (a.k + 7) / 8, total = a.top_k * k8;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  griddep_wait();
  griddep_launch();
  if ((int)threadIdx.x < a.top_k) s_ids[threadIdx.x] = __ldcg(a.ids + threadIdx.x);
  for (int j = 0; j < a.top_k; ++j) {
    const float p = __ldcg(a.probs + j);
    for (int c = threadIdx.x; c < k8 * 8; c += kStepThreads)
      hs[plane_at(j * k8 * 8 + c, total)] = c < a.k ? __ldcg(a.act + (size_t)j * a.k + c) * p : 0.f;
  }
  __syncthreads();
  for (int row0 = (blockIdx.x * 8 + warp) * RU; row0 < a.n; row0 += gridDim.x * 8 * RU) {
    float acc[RU];
#pragma unroll
    for (int i = 0; i < RU; ++i) acc[i] = 0.f;
#pragma unroll 1
    for (int j = 0; j < a.top_k; ++j) {
      const uint4* base = reinterpret_cast<const uint4*>(a.w + s_ids[j] * a.w_gstride + (long long)row0 * a.w_ld);
      const int ld8 = (int)(a.w_ld / 8);
#pragma unroll 1
      for (int c0 = lane; c0 < k8; c0 += 32 * U) {
        uint4 wv[RU][U];
#pragma unroll
        for (int q = 0; q < U; ++q)
#pragma unroll
          for (int i = 0; i < RU; ++i)
            wv[i][q] = c0 + q * 32 < k8 && row0 + i < a.n ? ld_stream(base + i * ld8 + c0 + q * 32) : make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
        for (int q = 0; q < U; ++q) {
          const int c = c0 + q * 32;
          if (c < k8) {
            const float4 x0 = hs4[j * k8 + c], x1 = hs4[total + j * k8 + c];
#pragma unroll
            for (int i = 0; i < RU; ++i) acc[i] = dot8(wv[i][q], x0, x1, acc[i]);
          }
        }
      }
    }
    __syncwarp();
#pragma unroll
    for (int i = 0; i < RU; ++i) {
      const float v = lane_sum(acc[i]);
      if (lane == 0 && row0 + i < a.n) a.out[row0 + i] = v;
    }
  }
}

int lanes_of(int k8) {
  int G = 4;
  while (G < 32 && G < k8) G *= 2;
  return G;
}

template <int PRO, int EPI, int RU, int U, bool ROUTE>
struct StepLaunch {
  // CTAs of this kernel that are resident at once with `smem` bytes each
  static int resident(size_t smem) {
    static size_t seen[8];
    static int value[8], count = 0;
    for (int i = 0; i < count; ++i)
      if (seen[i] == smem) return value[i];
    auto* kern = stack_step_kernel<PRO, EPI, RU, U, ROUTE>;
    if (count == 0 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxStepSmem) != cudaSuccess) return -1;
    int per = 0, dev = 0, sms = 148;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    if (cudaOccupancyMaxActiveBlocksPerMultiprocessor(&per, kern, kStepThreads, smem) != cudaSuccess || per < 1) per = 1;
    if (count < 8) { seen[count] = smem; value[count] = per * sms; ++count; }
    return per * sms;
  }
  static long long tiles(const StepArgs& a) {
    const int rows_tile = kStepThreads / lanes_of((a.k + 7) / 8) * RU;
    return (long long)a.groups * ((a.n + rows_tile - 1) / rows_tile);
  }
  static double balance(const StepArgs& a) {            // busy share of the resident CTAs
    const long long t = tiles(a), res = resident((size_t)((a.k + 7) / 8) * 32);
    if (res < 1) return 0.0;
    const long long grid = t < res ? t : res, per = (t + grid - 1) / grid;
    return (double)t / (double)(per * res);
  }
  static int run(const StepArgs& a, const RouterArgs& r, int groups, int keep, cudaStream_t stream, bool pdl) {
    const int k8 = (a.k + 7) / 8;
    const size_t smem = (size_t)k8 * 32;
    const long long t = tiles(a);
    if (smem > kMaxStepSmem || t < 1 || t > 0x7fffffffLL) return -7;
    const int res = resident(smem);
    if (res < 1) return -8;
    return launch_pdl(stack_step_kernel<PRO, EPI, RU, U, ROUTE>, dim3((unsigned)(t < res ? t : res)), dim3(kStepThreads), smem, stream, pdl, a,
                      r, groups, keep, lanes_of(k8));
  }
};

// Rows per lane group: the largest count that still spreads the rows evenly over the resident CTAs.
template <int PRO, int EPI, bool ROUTE>
int pick_step(const StepArgs& a, const RouterArgs& r, int groups, int keep, cudaStream_t stream, bool pdl) {
  if constexpr (EPI == kTEpiGlu || EPI == kTEpiRecur) {
    using A = StepLaunch<PRO, EPI, 2, 2, ROUTE>;
    using B = StepLaunch<PRO, EPI, 1, 4, ROUTE>;
    return A::balance(a) + 0.05 >= B::balance(a) ? A::run(a, r, groups, keep, stream, pdl) : B::run(a, r, groups, keep, stream, pdl);
  } else {
    using A = StepLaunch<PRO, EPI, 2, 4, ROUTE>;
    using B = StepLaunch<PRO, EPI, 1, 8, ROUTE>;
    return A::balance(a) + 0.05 >= B::balance(a) ? A::run(a, r, groups, keep, stream, pdl) : B::run(a, r, groups, keep, stream, pdl);
  }
}

}  // namespace

extern "C" int nrt_step_args_size() { return (int)sizeof(StepArgs); }
extern "C" int nrt_step_down_args_size() { return (int)sizeof(StepDownArgs); }

// `router` (expert form of the two-product epilogue): RouterArgs with the token's filled score row; the selection runs in every
// CTA and CTA 0 publishes it.
extern "C" int nrt_stack_step(int pro, int epi, const void* args, const void* router, int groups, int keep, void* stream, int pdl) {
  StepArgs a;
  memcpy(&a, args, sizeof(a));
  RouterArgs r;
  memset(&r, 0, sizeof(r));
  if (router) memcpy(&r, router, sizeof(r));
  if (a.n < 1 || a.k < 1 || a.groups < 1 || a.w_ld % 8 || a.w_gstride % 8 || a.w2_gstride % 8) return -3;
  if (router && (r.experts > 256 || r.top_k > 32 || r.rows != 1 || groups < 1 || groups > 32 || r.experts % groups)) return -3;
  if (epi == kTEpiConv && (a.hist_rows < 1 || a.hist_rows < 2 * (a.taps - 1) || a.groups != 1)) return -3;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const bool p = pdl != 0;
#define NRT_CASE(P, E) \
  if (pro == P && epi == E && !router) return pick_step<P, E, false>(a, r, groups, keep, s, p);
  NRT_CASE(kProResidual, kTEpiStore)
  NRT_CASE(kProResidual, kTEpiConv)
  NRT_CASE(kProResidual, kTEpiGlu)
  NRT_CASE(kProNorm, kTEpiStore)
  NRT_CASE(kProLoad, kTEpiStore)
  NRT_CASE(kProMerge, kTEpiGate)
  NRT_CASE(kProLoad, kTEpiRecur)
#undef NRT_CASE
  if (pro == kProNorm && epi == kTEpiGlu && router) return pick_step<kProNorm, kTEpiGlu, true>(a, r, groups, keep, s, p);
  return -2;
}

extern "C" int nrt_stack_down(const void* args, void* stream, int pdl) {
  StepDownArgs a;
  memcpy(&a, args, sizeof(a));
  if (a.n < 1 || a.k < 1 || a.top_k < 1 || a.top_k > 32 || a.w_ld % 8 || a.w_gstride % 8) return -3;
  const size_t smem = (size_t)a.top_k * ((a.k + 7) / 8) * 32;
  if (smem > kMaxStepSmem) return -7;
  auto run = [&](auto* kern, int ru) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxStepSmem);
    if (e != cudaSuccess) return (int)e;
    const int tiles = (a.n + 8 * ru - 1) / (8 * ru);
    return launch_pdl(kern, dim3(tiles < 592 ? tiles : 592), dim3(kStepThreads), smem, reinterpret_cast<cudaStream_t>(stream), pdl != 0, a);
  };
  if (a.n >= 8 * 2 * 296) return run(stack_down_kernel<2, 4>, 2);
  return run(stack_down_kernel<1, 8>, 1);
}
