// One-token step of layer stacks: matrix-vector products with their surroundings fused in.
//
// A single token reads every weight once, so the step is bound by HBM and the CUDA cores keep up with it; activations stay
// fp32 throughout.  Each launch is (prologue) -> W h -> (epilogue):
//   prologues  stream update + norms (every CTA repeats it: two row-sized L2 reads instead of a launch of its own), the same
//              with a mix of the previous token per group, norm of a segment, plain load per group, merge of the attention partials
//   epilogues  store / sigmoid / bias / squared relu, branches with the short convolution, output gate, two-product activations,
//              the recurrence step
// Weights stream through shared memory: each of the sixteen warps owns a run of output rows and a ring of its own (three 4 KiB
// slots) that one lane fills with bulk copies, so no two warps wait for one another inside the product.  The ring is filled
// before griddepcontrol.wait, where the choice of weights does not depend on the predecessor.  Measured on B200: smaller rings
// that let two kernels share an SM are slower (the successor's copies compete with the running product), and eight warps do not
// keep up with the copies.
#include "stack.cuh"
#include "launch.hpp"
#include "router.cuh"

#include <string.h>

using namespace nrt;

namespace {

constexpr int kStepThreads = 512;
constexpr int kPreN = 4096 / (kStepThreads * 4);       // float4 values per thread that cover the first 4096 elements

// The input vector lives in shared memory as two planes of float4: chunk c of eight elements is plane0[c], plane1[c], so that
// neighbouring lanes read neighbouring 16-byte words.
__device__ __forceinline__ int plane_at(int c, int k8) { return ((c >> 2) & 1) * k8 * 4 + (c >> 3) * 4 + (c & 3); }

__device__ __forceinline__ float dot8(const uint4& w, const float4& a, const float4& b, float acc) {
  float t = bf16_lo(w.z) * b.x;                  // two chains
  acc = fmaf(bf16_lo(w.x), a.x, acc);
  t = fmaf(bf16_hi(w.z), b.y, t);
  acc = fmaf(bf16_hi(w.x), a.y, acc);
  t = fmaf(bf16_lo(w.w), b.z, t);
  acc = fmaf(bf16_lo(w.y), a.z, acc);
  t = fmaf(bf16_hi(w.w), b.w, t);
  acc = fmaf(bf16_hi(w.y), a.w, acc);
  return acc + t;
}
// untiled bulk copy of weights that are read once per step (16-byte addresses and size)
__device__ __forceinline__ void bulk_load(void* dst, const void* src, uint32_t bytes, uint64_t* bar, uint64_t policy) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes.L2::cache_hint [%0], [%1], %2, [%3], %4;"
               ::"r"(smem_u32(dst)), "l"(src), "r"(bytes), "r"(smem_u32(bar)), "l"(policy)
               : "memory");
}

// Values of the first kPreSpan elements that do not depend on the predecessor kernel, requested before the wait for it: the
// norm weights, and the stream itself (written at least two launches back).
constexpr int kPreSpan = kStepThreads * 4 * kPreN;
struct Pre {
  float4 x[kPreN];
  uint2 post[kPreN], in[kPreN];
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
  for (int i = 0; i < kPreN; ++i) {
    const int e = (i * kStepThreads + (int)threadIdx.x) * 4;
    p.x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    p.post[i] = p.in[i] = make_uint2(0u, 0u);
    if (e < a.k) {
      if (a.in_w) p.in[i] = ldw4(a.in_w + e);
      if (PRO == kProResidual || PRO == kProMix) {
        if (a.y) p.post[i] = ldw4(a.post_w + e);
        if (!a.tokens) p.x[i] = ldcg4(a.x + e);
      }
    }
  }
}

__device__ __forceinline__ float sum4(const float4& v) { return (v.x + v.y) + (v.z + v.w); }
__device__ __forceinline__ float4 minus4(const float4& v, float m) { return make_float4(v.x - m, v.y - m, v.z - m, v.w - m); }
__device__ __forceinline__ float4 scale4(const float4& v, float s) { return make_float4(v.x * s, v.y * s, v.z * s, v.w * s); }
__device__ __forceinline__ float4 add4(const float4& a, const float4& b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }

// The input of one group in shared memory.  `slot`: state slot of the previous token (kProMix).
template <int PRO>
__device__ __forceinline__ void load_input(const StepArgs& a, int g, int k8, float* hs, float* red, const Pre& p, int pos, int slot) {
  const int K = a.k;
  float4* hs4 = reinterpret_cast<float4*>(hs);
  // element e (a multiple of four) of the input -> its float4 in the two planes
  auto at4 = [&](int e) -> float4& { return hs4[((e >> 2) & 1) * k8 + (e >> 3)]; };
  if (PRO == kProResidual || PRO == kProNorm || PRO == kProMix) {
    constexpr bool STREAM = PRO != kProNorm;
    const bool layer = STREAM && a.norm == kNormLayer;
    const __nv_bfloat16* emb = nullptr;
    if (STREAM && a.tokens) {
      int t = *reinterpret_cast<const volatile int*>(a.tokens);
      t = t < 0 ? 0 : t >= a.vocab ? a.vocab - 1 : t;
      emb = a.table + (size_t)t * K;
    }
    // kProMix: the previous token's stream (none at position 0), this group's mixing weights
    const float* before = PRO == kProMix && pos > 0 && slot >= 0 ? a.shift + (long long)slot * a.state_stride : nullptr;
    float* after = PRO == kProMix && blockIdx.x == 0 && slot >= 0 ? a.shift + (long long)(1 - slot) * a.state_stride : nullptr;
    const __nv_bfloat16* mu = PRO == kProMix ? a.mu + (long long)g * K : nullptr;
    if ((K & 3) == 0) {
      // the first kPreSpan elements stay in registers, the others in the input's own place
      float4 v[kPreN];
      auto each = [&](auto&& f) {
#pragma unroll
        for (int i = 0; i < kPreN; ++i) {
          const int e = (i * kStepThreads + (int)threadIdx.x) * 4;
          if (e < K) f(e, v[i]);
        }
        for (int e = kPreSpan + (int)threadIdx.x * 4; e < K; e += kStepThreads * 4) f(e, at4(e));
      };
      float mean = 0.f, r = 0.f;
      auto norm_of = [&](float part) {                   // sums of squares, or (layer norm) of values
        float sq = block_sum_f(part, red);
        mean = 0.f;
        if (layer) {
          mean = sq / (float)K;
          float d = 0.f;
          each([&](int, float4& t) { d += dot4(minus4(t, mean)); });
          sq = block_sum_f(d, red);
        }
        r = 1.0f / sqrtf(sq / (float)K + a.eps);
      };
      float part = 0.f;
      if (PRO == kProNorm) {
        each([&](int e, float4& t) { t = ldcg4(a.in_ + e); part += dot4(t); });
      } else {
        if (a.y) {
          if (a.y2) {
            // two branches: the mean of both, scaled to unit RMS
            float s1 = 0.f, s2 = 0.f;
            each([&](int e, float4& t) { t = ldcg4(a.y + e); s1 += dot4(t); s2 += dot4(ldcg4(a.y2 + e)); });
            const float r1 = 0.5f / sqrtf(block_sum_f(s1, red) / (float)K + a.eps), r2 = 0.5f / sqrtf(block_sum_f(s2, red) / (float)K + a.eps);
            each([&](int e, float4& t) {
              t = fma4(t, bf4(ldw4(a.join_w + e)), r1, fma4(ldcg4(a.y2 + e), bf4(ldw4(a.join_w2 + e)), r2, make_float4(0.f, 0.f, 0.f, 0.f)));
              part += layer ? sum4(t) : dot4(t);
            });
          } else {
            each([&](int e, float4& t) { t = ldcg4(a.y + e); part += layer ? sum4(t) : dot4(t); });
          }
          norm_of(part);
        }
        part = 0.f;
        auto stream = [&](int e, float4& t, float4 x, const float4& w) {
          if (emb) x = scale4(bf4(ldw4(emb + e)), a.embed_scale);
          if (a.y) x = fma4(minus4(t, mean), w, r, x);
          if (a.add) x = add4(x, bf4(ldw4(a.add + e)));
          if (blockIdx.x == 0) *reinterpret_cast<float4*>(a.x_out + e) = x;
          t = x;
          part += layer ? sum4(x) : dot4(x);
        };
#pragma unroll
        for (int i = 0; i < kPreN; ++i) {
          const int e = (i * kStepThreads + (int)threadIdx.x) * 4;
          if (e < K) stream(e, v[i], p.x[i], bf4(p.post[i]));
        }
        for (int e = kPreSpan + (int)threadIdx.x * 4; e < K; e += kStepThreads * 4)
          stream(e, at4(e), emb ? make_float4(0.f, 0.f, 0.f, 0.f) : ldcg4(a.x + e), a.y ? bf4(ldw4(a.post_w + e)) : make_float4(0.f, 0.f, 0.f, 0.f));
      }
      if (PRO == kProMix) {
        each([&](int e, float4& t) {
          if (after) *reinterpret_cast<float4*>(after + e) = t;
          const float4 b = before ? ldcg4(before + e) : make_float4(0.f, 0.f, 0.f, 0.f), m = bf4(ldw4(mu + e));
          at4(e) = make_float4(fmaf(b.x - t.x, m.x, t.x), fmaf(b.y - t.y, m.y, t.y), fmaf(b.z - t.z, m.z, t.z), fmaf(b.w - t.w, m.w, t.w));
        });
      } else if (STREAM && a.raw_in) {
        each([&](int e, float4& t) { at4(e) = t; });
      } else {
        norm_of(part);
        const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int i = 0; i < kPreN; ++i) {
          const int e = (i * kStepThreads + (int)threadIdx.x) * 4;
          if (e < K) at4(e) = fma4(minus4(v[i], mean), bf4(p.in[i]), r, zero);
        }
        for (int e = kPreSpan + (int)threadIdx.x * 4; e < K; e += kStepThreads * 4) at4(e) = fma4(minus4(at4(e), mean), bf4(ldw4(a.in_w + e)), r, zero);
      }
    } else {
      auto at = [&](int c) -> float& { return hs[plane_at(c, k8)]; };
      float mean = 0.f, r = 0.f;
      auto norm_of = [&]() {
        float part = 0.f;
        for (int c = threadIdx.x; c < K; c += kStepThreads) part += layer ? at(c) : at(c) * at(c);
        float sq = block_sum_f(part, red);
        mean = 0.f;
        if (layer) {
          mean = sq / (float)K;
          float d = 0.f;
          for (int c = threadIdx.x; c < K; c += kStepThreads) d = fmaf(at(c) - mean, at(c) - mean, d);
          sq = block_sum_f(d, red);
        }
        r = 1.0f / sqrtf(sq / (float)K + a.eps);
      };
      if (STREAM && a.y) {
        float r1 = 1.f, r2 = 0.f;
        if (a.y2) {
          float s1 = 0.f, s2 = 0.f;
          for (int c = threadIdx.x; c < K; c += kStepThreads) {
            const float t = __ldcg(a.y + c), u = __ldcg(a.y2 + c);
            s1 = fmaf(t, t, s1);
            s2 = fmaf(u, u, s2);
          }
          r1 = 0.5f / sqrtf(block_sum_f(s1, red) / (float)K + a.eps);
          r2 = 0.5f / sqrtf(block_sum_f(s2, red) / (float)K + a.eps);
        }
        for (int c = threadIdx.x; c < K; c += kStepThreads)
          at(c) = a.y2 ? __ldcg(a.y + c) * r1 * bf(a.join_w + c) + __ldcg(a.y2 + c) * r2 * bf(a.join_w2 + c) : __ldcg(a.y + c);
        norm_of();
      }
      for (int c = threadIdx.x; c < K; c += kStepThreads) {
        float x = PRO == kProNorm ? __ldcg(a.in_ + c) : emb ? bf(emb + c) * a.embed_scale : __ldcg(a.x + c);
        if (STREAM) {
          if (a.y) x += (at(c) - mean) * r * bf(a.post_w + c);
          if (a.add) x += bf(a.add + c);
          if (blockIdx.x == 0) a.x_out[c] = x;
        }
        if (PRO == kProMix) {
          if (after) after[c] = x;
          x = fmaf((before ? __ldcg(before + c) : 0.f) - x, bf(mu + c), x);
        }
        at(c) = x;
      }
      if (PRO == kProNorm || (PRO == kProResidual && !a.raw_in)) {
        norm_of();
        for (int c = threadIdx.x; c < K; c += kStepThreads) at(c) = (at(c) - mean) * r * bf(a.in_w + c);
      }
    }
  } else if (PRO == kProLoad) {
    const float* in = a.in_ + g * a.in_gstride;
    if (((K | (int)a.in_gstride) & 3) == 0) {
#pragma unroll 4
      for (int e = (int)threadIdx.x * 4; e < K; e += kStepThreads * 4) at4(e) = ldcg4(in + e);
    } else {
      for (int c = threadIdx.x; c < K; c += kStepThreads) hs[plane_at(c, k8)] = __ldcg(in + c);
    }
  } else if (PRO == kProExperts) {
    const int total = a.segs * k8;
    for (int j = 0; j < a.segs; ++j) {
      const float pj = __ldcg(a.probs + j);
      for (int c = threadIdx.x; c < k8 * 8; c += kStepThreads)
        hs[plane_at(j * k8 * 8 + c, total)] = c < K ? __ldcg(a.in_ + (size_t)j * K + c) * pj : 0.f;
    }
    __syncthreads();
    return;
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
    if ((int)threadIdx.x < used) ws[threadIdx.x] = w / l;           // used <= kMaxSplits <= threads
    int cols = 1;
    while (cols < k4 && cols < kStepThreads) cols *= 2;         // (both powers of two)
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
    v = row >= a.sig_from ? sigmoid_f(v) : v * a.scale;
    a.out[at] = a.bias ? v + bf(a.bias + at) : v;
  } else if (EPI == kTEpiRelu2) {
    a.out[at] = relu2_f(v);
  } else if (EPI == kTEpiConvSilu) {
    if (row < a.conv_rows) {
      float u = 0.f;
      for (int j = 0; j < a.taps - 1; ++j) {
        const int back = a.taps - 1 - j;
        if (back <= pos) u = fmaf(bf(a.conv + (size_t)row * a.taps + j), a.history[(long long)((pos - back) % a.hist_rows) * a.conv_rows + row], u);
      }
      u = fmaf(bf(a.conv + (size_t)row * a.taps + a.taps - 1), v, u);
      a.history[(long long)(pos % a.hist_rows) * a.conv_rows + row] = v;
      v = silu_f(u);
    }
    a.out[at] = v;
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

constexpr int kWarps = kStepThreads / 32;
constexpr int kSlot = 4096;                   // bytes of one ring slot of a warp
constexpr int kMaxStepSmem = 225 * 1024;

// How a launch cuts its rows: host-computed, the same for every CTA.
struct StepShape {
  int k8;            // 16-byte pieces of a row (per expert)
  int per_seg;       // slots of one row of one expert
  int rows_slot;     // > 0: short rows, this many per slot (row-block form)
  int G;             // lanes per row of the row-block form
  int q, units, parts;   // rows per unit, units, units per group (per-group inputs)
  int slots;         // ring slots per warp
};

template <int PRO, int EPI, bool ROUTE>
__global__ void __launch_bounds__(kStepThreads, 2) stack_step_kernel(const StepArgs a, const RouterArgs ra, const int rgroups,
                                                                     const int rkeep, const StepShape sh) {
  constexpr bool DUAL = EPI == kTEpiGlu || EPI == kTEpiRecur;
  constexpr bool PER_GROUP = PRO == kProLoad || PRO == kProMerge || PRO == kProMix;
  constexpr int CUT = DUAL ? kSlot / 32 : kSlot / 16;                  // pieces per slot and matrix
  extern __shared__ __align__(128) uint8_t dyn[];
  __shared__ float red[33];
  __shared__ int s_ids[32];
  __shared__ uint64_t bars[kWarps * 3];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  uint8_t* ring = dyn + warp * sh.slots * kSlot;
  float* hs = reinterpret_cast<float*>(dyn + kWarps * sh.slots * kSlot);
  const float4* hs4 = reinterpret_cast<const float4*>(hs);
  uint64_t* bar = bars + warp * 3;
  const int k8 = sh.k8, ld8 = (int)(a.w_ld / 8), total = a.segs * k8;
  const int n_last = a.n_last ? a.n_last : a.n, R = (a.groups - 1) * a.n + n_last;
  if (lane == 0) {
    for (int i = 0; i < sh.slots; ++i) mbar_init(&bar[i], 1);
    mbar_fence_init();
  }
  __syncwarp();
  const uint64_t policy = l2_policy_evict_first();

  // this warp's rows of a unit; the request cursor runs ahead of the consuming one by up to `slots`
  int w_end = 0, i_row = 0, i_seg = 0, i_sub = 0, i_slot = 0, issued = 0, used = 0;
  auto group_of = [&](int row) { return a.groups == 1 ? 0 : row / a.n; };
  auto rows_at = [&](int row) { return min(min(sh.rows_slot, w_end - row), a.n * (group_of(row) + 1) - row); };
  auto open_unit = [&](int u) {
    int lo, hi;
    if (PER_GROUP) {
      const int g = min(u / sh.parts, a.groups - 1), part = u - g * sh.parts, ng = g == a.groups - 1 ? n_last : a.n;
      lo = g * a.n + min(ng, part * sh.q);
      hi = g * a.n + min(ng, (part + 1) * sh.q);
    } else {
      lo = min(R, u * sh.q);
      hi = min(R, lo + sh.q);
    }
    const int per = (hi - lo + kWarps - 1) / kWarps;
    i_row = min(hi, lo + warp * per);
    w_end = min(hi, i_row + per);
    i_seg = i_sub = 0;
    return i_row;
  };
  auto request = [&]() {
    const int slot = i_slot, g = group_of(i_row), r = i_row - g * a.n;
    uint8_t* dst = ring + slot * kSlot;
    long long off;
    int count, rows = 1, wg = ROUTE ? s_ids[g] : PRO == kProExperts ? s_ids[0] : g;
    if (sh.rows_slot > 0) {
      rows = rows_at(i_row);
      count = rows * ld8;
      off = (long long)r * a.w_ld;
    } else {
      if (PRO == kProExperts) wg = s_ids[i_seg];
      count = min(CUT, k8 - i_sub * CUT);
      off = (long long)r * a.w_ld + i_sub * CUT * 8;
    }
    if (lane == 0) {
      mbar_expect_tx(&bar[slot], (DUAL ? 2u : 1u) * count * 16u);
      bulk_load(dst, a.w + wg * a.w_gstride + off, count * 16u, &bar[slot], policy);
      if (DUAL) bulk_load(dst + CUT * 16, a.w2 + wg * a.w2_gstride + off, count * 16u, &bar[slot], policy);
    }
    ++issued;
    if (++i_slot == sh.slots) i_slot = 0;
    if (sh.rows_slot > 0) i_row += rows;
    else if (++i_sub == sh.per_seg) {
      i_sub = 0;
      if (++i_seg == a.segs) { i_seg = 0; ++i_row; }
    }
  };
  auto fill = [&]() {
    while (i_row < w_end && issued - used < sh.slots) request();
  };

  int unit = blockIdx.x;
  int row = open_unit(unit);
  constexpr bool EARLY = !ROUTE && PRO != kProExperts;                 // which weights is known before the predecessor ends
  if (EARLY) fill();
  Pre pre;
  if constexpr (PRO == kProResidual || PRO == kProMix) preload<PRO>(a, pre);   // (a normed input may come from the predecessor itself)
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
  if (PRO == kProExperts) {
    if ((int)threadIdx.x < a.segs) s_ids[threadIdx.x] = __ldcg(a.ids + threadIdx.x);
    __syncthreads();
  }
  if (!EARLY) fill();
  int slot = 1;
  if (EPI == kTEpiRecur || PRO == kProMix) slot = state_slot(a.tags, pos, a.status);
  if constexpr (PRO == kProNorm) preload<PRO>(a, pre);
  if (!PER_GROUP) load_input<PRO>(a, 0, k8, hs, red, pre, pos, slot);
  if (PRO == kProNorm && a.lat_in && blockIdx.x == gridDim.x - 1 && pos >= 0 && pos < a.capacity) {
    // append the token's key/value latent to the cache
    float sq = 0.f;
    for (int c = threadIdx.x; c < a.lat_rank; c += kStepThreads) { const float v = __ldcg(a.lat_in + c); sq = fmaf(v, v, sq); }
    const float rs = 1.0f / sqrtf(block_sum_f(sq, red) / (float)a.lat_rank + a.eps);
    for (int c = threadIdx.x; c < a.lat_rank; c += kStepThreads)
      store_act(a.lat_cache, (long long)pos * a.lat_ld + c, __ldcg(a.lat_in + c) * rs * bf(a.lat_w + c), a.f32);
  }

  bool ok = true;
  int u_slot = 0;
  uint32_t u_phase = 0;
  while (true) {
    if (PER_GROUP) load_input<PRO>(a, min(unit / sh.parts, a.groups - 1), k8, hs, red, pre, pos, slot);
    // results of up to 32 finished rows wait in the lanes, then all lanes run the epilogue at once
    float acc = 0.f, acc2 = 0.f, res = 0.f, res2 = 0.f;
    int ready = 0, first = row, seg = 0, sub = 0;
    auto flush = [&]() {
      if (lane < ready && slot >= 0) {
        const int at = first + lane, g = group_of(at);
        finish_row<EPI>(a, g, at - g * a.n, res, res2, pos, slot);
      }
      first += ready;
      ready = 0;
      __syncwarp();
    };
    while (row < w_end && ok) {
      const int s = u_slot;
      ok = __all_sync(0xffffffffu, mbar_wait(&bar[s], u_phase, a.status, kSiteTmaFull | (warp & 7)));
      if (!ok) break;
      const uint4* w0 = reinterpret_cast<const uint4*>(ring + s * kSlot);
      const uint4* w1 = w0 + CUT;
      if (sh.rows_slot > 0) {
        const int rows = rows_at(row), lig = lane & (sh.G - 1), mine = lane / sh.G, per = 32 / sh.G;
        if (ready + rows > 32) flush();
        for (int r0 = 0; r0 < rows; r0 += per) {
          const int rr = r0 + mine;
          float v = 0.f, v2 = 0.f;
          if (rr < rows)
            for (int c = lig; c < k8; c += sh.G) {
              const float4 x0 = hs4[c], x1 = hs4[total + c];
              v = dot8(w0[rr * ld8 + c], x0, x1, v);
              if (DUAL) v2 = dot8(w1[rr * ld8 + c], x0, x1, v2);
            }
          for (int o = sh.G >> 1; o > 0; o >>= 1) {
            v += __shfl_xor_sync(0xffffffffu, v, o);
            if (DUAL) v2 += __shfl_xor_sync(0xffffffffu, v2, o);
          }
          const int want = lane - (ready + r0);                        // row of this pass that belongs to this lane
          const int src = (want * sh.G) & 31;
          const float t = __shfl_sync(0xffffffffu, v, src), t2 = DUAL ? __shfl_sync(0xffffffffu, v2, src) : 0.f;
          if (want >= 0 && want < per && r0 + want < rows) { res = t; res2 = t2; }
        }
        ready += rows;
        row += rows;
      } else {
        const int count = min(CUT, k8 - sub * CUT);
        const float4* h0 = hs4 + seg * k8 + sub * CUT;
        const float4* h1 = h0 + total;
#pragma unroll
        for (int i = 0; i < CUT / 32; ++i) {
          const int c = lane + 32 * i;
          if (c < count) {
            const float4 x0 = h0[c], x1 = h1[c];
            acc = dot8(w0[c], x0, x1, acc);
            if (DUAL) acc2 = dot8(w1[c], x0, x1, acc2);
          }
        }
        if (++sub == sh.per_seg) { sub = 0; ++seg; }
        if (seg == a.segs) {
          seg = 0;
          const float v = lane_sum(acc), v2 = DUAL ? lane_sum(acc2) : 0.f;
          acc = acc2 = 0.f;
          if (lane == ready) { res = v; res2 = v2; }
          ++row;
          if (++ready == 32) flush();
        }
      }
      ++used;
      if (++u_slot == sh.slots) { u_slot = 0; u_phase ^= 1; }
      __syncwarp();                                                    // every lane has read the slot before it is requested anew
      fill();
    }
    flush();
    unit += gridDim.x;
    if (unit >= sh.units) break;
    row = open_unit(unit);
    if (ok) fill();
    __syncthreads();                                                   // the input vector is replaced
  }
  // A CTA that starts after this store still finds `pos` in its own slot: only the other slot's tag changes.
  if (EPI == kTEpiRecur && slot >= 0 && blockIdx.x == 0 && threadIdx.x == 0) {
    a.tags[1 - slot] = pos + 1;
    if (pos == 0) a.tags[1] = -1;
  }
  if (!ok) drain_on_error(a.status);
}

int step_sms() {
  static int sms = 0;
  if (!sms) {
    int dev = 0;
    cudaGetDevice(&dev);
    if (cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || sms < 1) sms = 148;
  }
  return sms;
}

template <int PRO, int EPI, bool ROUTE>
int launch_step(const StepArgs& a, const RouterArgs& r, int groups, int keep, cudaStream_t stream, bool pdl) {
  constexpr bool DUAL = EPI == kTEpiGlu || EPI == kTEpiRecur;
  constexpr bool PER_GROUP = PRO == kProLoad || PRO == kProMerge || PRO == kProMix;
  constexpr int CUT = DUAL ? kSlot / 32 : kSlot / 16;
  auto* kern = stack_step_kernel<PRO, EPI, ROUTE>;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxStepSmem - (ROUTE ? 8192 : 0));
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const int n_last = a.n_last ? a.n_last : a.n;
  const long long R = (long long)(a.groups - 1) * a.n + n_last;
  if (R > 0x7fffffffLL) return -3;
  StepShape s = {};
  s.k8 = (a.k + 7) / 8;
  const int ld8 = (int)(a.w_ld / 8);
  if (a.segs == 1 && ld8 * 2 <= CUT) {                   // short rows travel in blocks
    s.rows_slot = CUT / ld8 < 32 ? CUT / ld8 : 32;
    s.G = 1;
    while (s.G < 32 && s.G < s.k8) s.G *= 2;
  } else {
    s.per_seg = (s.k8 + CUT - 1) / CUT;
  }
  const int sms = step_sms();
  if (PER_GROUP) {
    // the most parts per group (a shorter last group gets fewer) that fill the SMs once
    auto last = [&]() { return (n_last + s.q - 1) / s.q; };
    s.parts = n_last < a.n && a.groups > 1 ? sms / (a.groups - 1) : sms / a.groups;
    for (s.parts = s.parts > 1 ? s.parts : 1;; --s.parts) {
      s.q = (a.n + s.parts - 1) / s.parts;
      if (s.parts == 1 || (a.groups - 1) * ((a.n + s.q - 1) / s.q) + last() <= sms) break;
    }
    s.parts = (a.n + s.q - 1) / s.q;
    s.units = (a.groups - 1) * s.parts + last();
  } else {
    const long long want = (R + kWarps - 1) / kWarps;
    const int grid = (int)(want < sms ? want : sms);
    s.q = (int)((R + grid - 1) / grid);
    s.units = (int)((R + s.q - 1) / s.q);
    s.parts = 1;
  }
  const int hs_bytes = a.segs * s.k8 * 32, limit = kMaxStepSmem - (ROUTE ? 8192 : 0);
  for (s.slots = 3; s.slots > 1 && kWarps * s.slots * kSlot + hs_bytes > limit; --s.slots) {}
  const int smem = kWarps * s.slots * kSlot + hs_bytes;
  if (smem > limit) return -7;
  return launch_pdl(kern, dim3(s.units < sms ? s.units : sms), dim3(kStepThreads), smem, stream, pdl, a, r, groups, keep, s);
}

}  // namespace

extern "C" int nrt_step_args_size() { return (int)sizeof(StepArgs); }

// `router` (expert form of the two-product epilogue): RouterArgs with the token's filled score row; the selection runs in every
// CTA and CTA 0 publishes it.
extern "C" int nrt_stack_step(int pro, int epi, const void* args, const void* router, int groups, int keep, void* stream, int pdl) {
  StepArgs a;
  memcpy(&a, args, sizeof(a));
  RouterArgs r;
  memset(&r, 0, sizeof(r));
  if (router) memcpy(&r, router, sizeof(r));
  if (a.n < 1 || a.k < 1 || a.groups < 1 || a.segs < 1 || a.segs > 32 || (a.segs > 1 && pro != kProExperts) || a.w_ld % 8 || a.w_gstride % 8 || a.w2_gstride % 8) return -3;
  if (router && (r.experts > 256 || r.top_k > 32 || r.rows != 1 || groups < 1 || groups > 32 || r.experts % groups)) return -3;
  if (a.n_last < 0 || a.n_last > a.n || (a.y2 && (!a.y || !a.join_w || !a.join_w2))) return -3;
  if ((pro == kProResidual || pro == kProMix) && a.y && !a.post_w) return -3;
  if (pro == kProResidual && !a.raw_in && !a.in_w) return -3;
  if (pro == kProMix && (!a.mu || !a.shift || !a.tags)) return -3;
  if (epi == kTEpiConvSilu && (a.hist_rows < 1 || a.hist_rows < 2 * (a.taps - 1) || a.groups != 1 || a.conv_rows > a.n)) return -3;
  if (epi == kTEpiConv && (a.hist_rows < 1 || a.hist_rows < 2 * (a.taps - 1) || a.groups != 1)) return -3;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const bool p = pdl != 0;
#define NRT_CASE(P, E) \
  if (pro == P && epi == E && !router) return launch_step<P, E, false>(a, r, groups, keep, s, p);
  NRT_CASE(kProResidual, kTEpiStore)
  NRT_CASE(kProResidual, kTEpiConv)
  NRT_CASE(kProResidual, kTEpiGlu)
  NRT_CASE(kProResidual, kTEpiConvSilu)
  NRT_CASE(kProResidual, kTEpiRelu2)
  NRT_CASE(kProMix, kTEpiStore)
  NRT_CASE(kProNorm, kTEpiStore)
  NRT_CASE(kProLoad, kTEpiStore)
  NRT_CASE(kProExperts, kTEpiStore)
  NRT_CASE(kProMerge, kTEpiGate)
  NRT_CASE(kProLoad, kTEpiRecur)
#undef NRT_CASE
  if (pro == kProNorm && epi == kTEpiGlu && router) return launch_step<kProNorm, kTEpiGlu, true>(a, r, groups, keep, s, p);
  return -2;
}
