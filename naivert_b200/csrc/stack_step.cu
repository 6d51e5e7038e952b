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

template <int PRO>
__device__ __forceinline__ void load_input(const StepArgs& a, int g, int k8, float* hs, float* red) {
  const int K = a.k;
  if (PRO == kProResidual) {
    float ss = 0.f;
    if (a.y) {
      for (int c = threadIdx.x; c < K; c += kStepThreads) { const float v = __ldcg(a.y + c); ss = fmaf(v, v, ss); }
      ss = block_sum_f(ss, red);
    }
    const float ry = a.y ? 1.0f / sqrtf(ss / (float)K + a.eps) : 0.f;
    const __nv_bfloat16* emb = nullptr;
    if (a.tokens) {
      int t = *a.tokens;
      t = t < 0 ? 0 : t >= a.vocab ? a.vocab - 1 : t;
      emb = a.table + (size_t)t * K;
    }
    float sq = 0.f;
    for (int c = threadIdx.x; c < K; c += kStepThreads) {
      float v = emb ? bf(emb + c) * a.embed_scale : __ldcg(a.x + c);
      if (a.y) v += __ldcg(a.y + c) * ry * bf(a.post_w + c);
      if (a.add) v += bf(a.add + c);
      hs[plane_at(c, k8)] = v;
      if (blockIdx.x == 0) a.x_out[c] = v;
      sq = fmaf(v, v, sq);
    }
    sq = block_sum_f(sq, red);
    const float rx = 1.0f / sqrtf(sq / (float)K + a.eps);
    for (int c = threadIdx.x; c < K; c += kStepThreads) hs[plane_at(c, k8)] *= rx * bf(a.in_w + c);
  } else if (PRO == kProNorm) {
    float sq = 0.f;
    for (int c = threadIdx.x; c < K; c += kStepThreads) {
      const float v = __ldcg(a.in_ + c);
      hs[plane_at(c, k8)] = v;
      sq = fmaf(v, v, sq);
    }
    sq = block_sum_f(sq, red);
    const float rx = 1.0f / sqrtf(sq / (float)K + a.eps);
    for (int c = threadIdx.x; c < K; c += kStepThreads) hs[plane_at(c, k8)] *= rx * bf(a.in_w + c);
  } else if (PRO == kProLoad) {
    const float* in = a.in_ + g * a.in_gstride;
    for (int c = threadIdx.x; c < K; c += kStepThreads) hs[plane_at(c, k8)] = __ldcg(in + c);
  } else {                                                             // kProMerge
    const size_t row = K + 2, hstride = (size_t)a.groups * row;
    const float* p0 = a.part + g * row;
    float m = -FLT_MAX, l = 0.f;
    for (int s = 0; s < a.splits; ++s) m = fmaxf(m, __ldcg(p0 + s * hstride));
    for (int s = 0; s < a.splits; ++s) l += __ldcg(p0 + s * hstride + 1) * expf(__ldcg(p0 + s * hstride) - m);
    const float inv = 1.0f / l;
    for (int c = threadIdx.x; c < K; c += kStepThreads) {
      float v = 0.f;
      for (int s = 0; s < a.splits; ++s) {
        const float ms = __ldcg(p0 + s * hstride);
        if (ms > -FLT_MAX) v = fmaf(__ldcg(p0 + s * hstride + 2 + c), expf(ms - m), v);
      }
      hs[plane_at(c, k8)] = v * inv;
    }
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
  if (!PER_GROUP) load_input<PRO>(a, 0, k8, hs, red);
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
      load_input<PRO>(a, g, k8, hs, red);
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
    for (int c0 = lane; c0 < total; c0 += 32 * U) {
      uint4 wv[RU][U];
#pragma unroll
      for (int q = 0; q < U; ++q) {
        const int c = c0 + q * 32;
        const int j = c / k8;
        const bool in = c < total;
        const __nv_bfloat16* base = a.w + (in ? s_ids[j] : 0) * a.w_gstride;
#pragma unroll
        for (int i = 0; i < RU; ++i)
          wv[i][q] = in && row0 + i < a.n ? ld_stream(reinterpret_cast<const uint4*>(base + (long long)(row0 + i) * a.w_ld) + (c - j * k8))
                                          : make_uint4(0u, 0u, 0u, 0u);
      }
#pragma unroll
      for (int q = 0; q < U; ++q) {
        const int c = c0 + q * 32;
        if (c < total) {
          const float4 x0 = hs4[c], x1 = hs4[total + c];
#pragma unroll
          for (int i = 0; i < RU; ++i) acc[i] = dot8(wv[i][q], x0, x1, acc[i]);
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

constexpr int kMaxStepSmem = 200 * 1024;

template <int PRO, int EPI, int RU, int U, bool ROUTE>
int launch_step(const StepArgs& a, const RouterArgs& r, int groups, int keep, cudaStream_t stream, bool pdl) {
  auto* kern = stack_step_kernel<PRO, EPI, RU, U, ROUTE>;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxStepSmem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const int k8 = (a.k + 7) / 8;
  int G = 4;
  while (G < 32 && G < k8) G *= 2;
  const int rows_tile = kStepThreads / G * RU;
  const long long tiles = (long long)a.groups * ((a.n + rows_tile - 1) / rows_tile);
  const size_t smem = (size_t)k8 * 32;
  if (smem > kMaxStepSmem || tiles < 1 || tiles > 0x7fffffffLL) return -7;
  const int cap = PRO == kProMerge ? 148 * 2 : 148 * 4;
  return launch_pdl(kern, dim3((unsigned)(tiles < cap ? tiles : cap)), dim3(kStepThreads), smem, stream, pdl, a, r, groups, keep, G);
}

// Rows per lane group: as many as still leave every SM two CTAs.
template <int PRO, int EPI, bool ROUTE>
int pick_step(const StepArgs& a, const RouterArgs& r, int groups, int keep, cudaStream_t stream, bool pdl) {
  const long long rows = (long long)a.groups * a.n;
  const int k8 = (a.k + 7) / 8;
  int G = 4;
  while (G < 32 && G < k8) G *= 2;
  const long long per = kStepThreads / G;
  if constexpr (EPI == kTEpiGlu || EPI == kTEpiRecur) {
    if (rows >= 2 * per * 296) return launch_step<PRO, EPI, 2, 2, ROUTE>(a, r, groups, keep, stream, pdl);
    return launch_step<PRO, EPI, 1, 4, ROUTE>(a, r, groups, keep, stream, pdl);
  } else {
    if (rows >= 4 * per * 296) return launch_step<PRO, EPI, 4, 2, ROUTE>(a, r, groups, keep, stream, pdl);
    if (rows >= 2 * per * 296) return launch_step<PRO, EPI, 2, 4, ROUTE>(a, r, groups, keep, stream, pdl);
    return launch_step<PRO, EPI, 1, 8, ROUTE>(a, r, groups, keep, stream, pdl);
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
