// Row kernels of layer stacks (chunk path): stream update + norms, latent preparation, short convolution, the gated
// linear recurrence as a chunked scan, and the expert row permutation.
#include "stack.cuh"
#include "launch.hpp"
#include "router.cuh"

#include <string.h>

using namespace nrt;

namespace {

// ------------------------------------------------------------------------------------ stream update + norms
// One CTA per row.  x (+ embedding) -> x += norm(y) * post_w + add -> h = norm(x) * pre_w (or x itself), all in float.
__device__ __forceinline__ float4 bf4(const __nv_bfloat16* p) {
  const uint2 v = __ldg(reinterpret_cast<const uint2*>(p));
  return make_float4(bf16_lo(v.x), bf16_hi(v.x), bf16_lo(v.y), bf16_hi(v.y));
}
__device__ __forceinline__ float dot4(const float4& v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
__device__ __forceinline__ float sum4(const float4& v) { return (v.x + v.y) + (v.z + v.w); }
__device__ __forceinline__ float4 minus4(const float4& v, float m) { return make_float4(v.x - m, v.y - m, v.z - m, v.w - m); }

// What a row is shifted and scaled by: `part` is the thread's sum of squares (RMS) or of values (layer norm: the squared
// deviations are summed in a second pass over the thread's own values, `again(mean)`).
struct RowNorm { float mean, r; };
template <class Again>
__device__ __forceinline__ RowNorm row_norm(int kind, float part, int width, float eps, float* red, Again again) {
  RowNorm n;
  n.mean = 0.f;
  float sq = block_sum_f(part, red);
  if (kind == kNormLayer) {
    n.mean = sq / (float)width;
    sq = block_sum_f(again(n.mean), red);
  }
  n.r = 1.0f / sqrtf(sq / (float)width + eps);
  return n;
}

// widths that are multiples of four: 16-byte accesses, several in flight per thread
__device__ __forceinline__ void rows_vec4(const StackRowArgs& a, int r, float4* buf, float* red) {
  const int W4 = a.width / 4;
  const bool layer = a.norm == kNormLayer;
  float4* sy = buf;
  float4* sx = buf + W4;
  RowNorm ny = {0.f, 0.f};
  float4* xrow = reinterpret_cast<float4*>(a.x + (size_t)r * a.width);
  if (a.y) {
    float ss = 0.f;
    if (a.slot_of) {
      for (int c = threadIdx.x; c < W4; c += 256) {
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int j = 0; j < a.top_k; ++j) {
          const float p = a.probs[(size_t)r * a.top_k + j];
          const float4 t = reinterpret_cast<const float4*>(a.y + (long long)a.slot_of[(size_t)r * a.top_k + j] * a.y_ld)[c];
          v = make_float4(fmaf(p, t.x, v.x), fmaf(p, t.y, v.y), fmaf(p, t.z, v.z), fmaf(p, t.w, v.w));
        }
        sy[c] = v;
        ss += layer ? sum4(v) : dot4(v);
      }
    } else if (a.y2) {
      const float4* y = reinterpret_cast<const float4*>(a.y + (long long)r * a.y_ld);
      const float4* y2 = reinterpret_cast<const float4*>(a.y2 + (long long)r * a.y_ld);
      float s1 = 0.f, s2 = 0.f;
#pragma unroll 4
      for (int c = threadIdx.x; c < W4; c += 256) {
        const float4 v = y[c], w = y2[c];
        sy[c] = v;
        sx[c] = w;
        s1 += dot4(v);
        s2 += dot4(w);
      }
      const float r1 = 0.5f / sqrtf(block_sum_f(s1, red) / (float)a.width + a.eps), r2 = 0.5f / sqrtf(block_sum_f(s2, red) / (float)a.width + a.eps);
#pragma unroll 4
      for (int c = threadIdx.x; c < W4; c += 256) {
        const float4 v = sy[c], w = sx[c], wv = bf4(a.join_w + c * 4), ww = bf4(a.join_w2 + c * 4);
        const float4 t = make_float4(fmaf(v.x * r1, wv.x, w.x * r2 * ww.x), fmaf(v.y * r1, wv.y, w.y * r2 * ww.y),
                                     fmaf(v.z * r1, wv.z, w.z * r2 * ww.z), fmaf(v.w * r1, wv.w, w.w * r2 * ww.w));
        sy[c] = t;
        ss += layer ? sum4(t) : dot4(t);
      }
    } else {
      const float4* y = reinterpret_cast<const float4*>(a.y + (long long)r * a.y_ld);
#pragma unroll 4
      for (int c = threadIdx.x; c < W4; c += 256) {
        const float4 v = y[c];
        sy[c] = v;
        ss += layer ? sum4(v) : dot4(v);
      }
    }
    ny = row_norm(a.norm, ss, a.width, a.eps, red, [&](float mean) {
      float sq = 0.f;
      for (int c = threadIdx.x; c < W4; c += 256) sq += dot4(minus4(sy[c], mean));
      return sq;
    });
  }
  const __nv_bfloat16* emb = nullptr;
  if (a.tokens) {
    int t = a.tokens[r];
    t = t < 0 ? 0 : t >= a.vocab ? a.vocab - 1 : t;
    emb = a.table + (size_t)t * a.width;
  }
  float part = 0.f;
#pragma unroll 4
  for (int c = threadIdx.x; c < W4; c += 256) {
    float4 v;
    if (emb) { v = bf4(emb + c * 4); v = make_float4(v.x * a.embed_scale, v.y * a.embed_scale, v.z * a.embed_scale, v.w * a.embed_scale); }
    else v = xrow[c];
    if (a.y) {
      const float4 y = minus4(sy[c], ny.mean), w = bf4(a.post_w + c * 4);
      v = make_float4(fmaf(y.x * ny.r, w.x, v.x), fmaf(y.y * ny.r, w.y, v.y), fmaf(y.z * ny.r, w.z, v.z), fmaf(y.w * ny.r, w.w, v.w));
    }
    if (a.add) { const float4 t = bf4(a.add + c * 4); v = make_float4(v.x + t.x, v.y + t.y, v.z + t.z, v.w + t.w); }
    xrow[c] = v;
    sx[c] = v;
    part += layer ? sum4(v) : dot4(v);
  }
  if (!a.pre_w && !a.copy_h) return;
  RowNorm nx = {0.f, 1.f};
  if (a.pre_w)
    nx = row_norm(a.norm, part, a.width, a.eps, red, [&](float mean) {
      float sq = 0.f;
      for (int c = threadIdx.x; c < W4; c += 256) sq += dot4(minus4(sx[c], mean));
      return sq;
    });
#pragma unroll 4
  for (int c = threadIdx.x; c < W4; c += 256) {
    float4 o = sx[c];
    if (a.pre_w) {
      const float4 v = minus4(o, nx.mean), w = bf4(a.pre_w + c * 4);
      o = make_float4(v.x * nx.r * w.x, v.y * nx.r * w.y, v.z * nx.r * w.z, v.w * nx.r * w.w);
    }
    if (a.h_f32) reinterpret_cast<float4*>(reinterpret_cast<float*>(a.h) + (long long)r * a.h_ld)[c] = o;
    else reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(a.h) + (long long)r * a.h_ld)[c] =
        make_uint2(pack_bf16x2(o.x, o.y), pack_bf16x2(o.z, o.w));
  }
}
__global__ void __launch_bounds__(256) stack_rows_kernel(const StackRowArgs a) {
  extern __shared__ __align__(16) float buf[];   // [2][width]: sublayer row, stream row
  __shared__ float red[33];
  griddep_wait();
  griddep_launch();
  const int r = blockIdx.x, W = a.width;
  if (((W | (int)a.y_ld | (int)a.h_ld) & 3) == 0) {
    rows_vec4(a, r, reinterpret_cast<float4*>(buf), red);
    return;
  }
  const bool layer = a.norm == kNormLayer;
  float* sy = buf;
  float* sx = buf + W;
  RowNorm ny = {0.f, 0.f};
  if (a.y) {
    float ss = 0.f;
    if (a.y2) {
      float s1 = 0.f, s2 = 0.f;
      for (int c = threadIdx.x; c < W; c += 256) {
        const float v = a.y[(long long)r * a.y_ld + c], w = a.y2[(long long)r * a.y_ld + c];
        sy[c] = v;
        sx[c] = w;
        s1 = fmaf(v, v, s1);
        s2 = fmaf(w, w, s2);
      }
      const float r1 = 0.5f / sqrtf(block_sum_f(s1, red) / (float)W + a.eps), r2 = 0.5f / sqrtf(block_sum_f(s2, red) / (float)W + a.eps);
      for (int c = threadIdx.x; c < W; c += 256) sy[c] = sy[c] * r1 * bf(a.join_w + c) + sx[c] * r2 * bf(a.join_w2 + c);
    } else if (a.slot_of) {
      for (int c = threadIdx.x; c < W; c += 256) {
        float v = 0.f;
        for (int j = 0; j < a.top_k; ++j)
          v = fmaf(a.probs[(size_t)r * a.top_k + j], a.y[(long long)a.slot_of[(size_t)r * a.top_k + j] * a.y_ld + c], v);
        sy[c] = v;
      }
    } else {
      for (int c = threadIdx.x; c < W; c += 256) sy[c] = a.y[(long long)r * a.y_ld + c];
    }
    for (int c = threadIdx.x; c < W; c += 256) ss += layer ? sy[c] : sy[c] * sy[c];
    ny = row_norm(a.norm, ss, W, a.eps, red, [&](float mean) {
      float sq = 0.f;
      for (int c = threadIdx.x; c < W; c += 256) sq = fmaf(sy[c] - mean, sy[c] - mean, sq);
      return sq;
    });
  }
  const __nv_bfloat16* emb = nullptr;
  if (a.tokens) {
    int t = a.tokens[r];
    t = t < 0 ? 0 : t >= a.vocab ? a.vocab - 1 : t;
    emb = a.table + (size_t)t * W;
  }
  float part = 0.f;
  for (int c = threadIdx.x; c < W; c += 256) {
    float v = emb ? bf(emb + c) * a.embed_scale : a.x[(size_t)r * W + c];
    if (a.y) v += (sy[c] - ny.mean) * ny.r * bf(a.post_w + c);
    if (a.add) v += bf(a.add + c);
    a.x[(size_t)r * W + c] = v;
    sx[c] = v;
    part += layer ? v : v * v;
  }
  if (!a.pre_w && !a.copy_h) return;
  RowNorm nx = {0.f, 1.f};
  if (a.pre_w)
    nx = row_norm(a.norm, part, W, a.eps, red, [&](float mean) {
      float sq = 0.f;
      for (int c = threadIdx.x; c < W; c += 256) sq = fmaf(sx[c] - mean, sx[c] - mean, sq);
      return sq;
    });
  for (int c = threadIdx.x; c < W; c += 256)
    store_act(a.h, (long long)r * a.h_ld + c, a.pre_w ? (sx[c] - nx.mean) * nx.r * bf(a.pre_w + c) : sx[c], a.h_f32);
}

// ------------------------------------------------------------------------------------ latent preparation
// grid (rows, 2): y = 0 normalises the query latent, y = 1 the key/value latent into its cache row.
__global__ void __launch_bounds__(256) latent_prep_kernel(const LatentPrepArgs a) {
  __shared__ float red[33];
  griddep_wait();
  griddep_launch();
  const int r = blockIdx.x, which = blockIdx.y;
  const int n = which ? a.kv_rank : a.q_rank;
  const float* src = a.proj + (long long)r * a.ld + (which ? a.q_rank : 0);
  const __nv_bfloat16* w = which ? a.kv_w : a.q_w;
  float ss = 0.f;
  for (int c = threadIdx.x; c < n; c += 256) ss = fmaf(src[c], src[c], ss);
  const float rs = 1.0f / sqrtf(block_sum_f(ss, red) / (float)n + a.eps);
  void* dst = which ? a.cache : a.cq;
  const int row = which ? *a.pos0 + r : r;
  if (which && (row < 0 || row >= a.capacity)) return;
  const long long base = (long long)row * (which ? a.cache_ld : a.cq_ld);
  for (int c = threadIdx.x; c < n; c += 256) store_act(dst, base + c, src[c] * rs * bf(w + c), a.f32);
}

// ------------------------------------------------------------------------------------ short convolution
// u[r][c] = b[c] + sum_j k[c][j] x[position of tap j], zeros before the sequence.  One thread owns a channel of a strip of
// rows; up to kConvWin taps stay in a register window, longer kernels re-read their inputs.
constexpr int kConvRows = 32, kConvWin = 4, kBatch = 8;

__device__ __forceinline__ float conv_input(const RecurrenceArgs& a, int r, int c, int pos0) {     // x at row r (negative: history)
  if (pos0 + r < 0) return 0.f;
  return r >= 0 ? load_act(a.xy, (long long)r * a.xy_ld + a.width + c, a.f32)
                : a.history[(long long)((pos0 + r) % a.hist_rows) * a.width + c];
}

__global__ void __launch_bounds__(128) stack_conv_kernel(const RecurrenceArgs a) {
  griddep_wait();
  griddep_launch();
  const int r0 = blockIdx.x * kConvRows, c = blockIdx.y * 128 + threadIdx.x;
  if (c >= a.width) return;
  const int pos0 = *a.pos0, rows = min(kConvRows, a.rows - r0);
  const int b = c / a.block;
  const long long u0 = ((long long)r0 * a.blocks + b) * a.block_pad + (c - b * a.block), ustep = (long long)a.blocks * a.block_pad;
  const float bias = bf(a.conv_b + c);
  if (a.taps <= kConvWin) {
    float k[kConvWin], x[kConvWin];                  // newest last; missing taps are zero
#pragma unroll
    for (int j = 0; j < kConvWin; ++j) {
      const int t = j - (kConvWin - a.taps);
      k[j] = t >= 0 ? bf(a.conv + (size_t)c * a.taps + t) : 0.f;
    }
#pragma unroll
    for (int j = 1; j < kConvWin; ++j) x[j] = j > kConvWin - a.taps ? conv_input(a, r0 - (kConvWin - j), c, pos0) : 0.f;
#pragma unroll 1
    for (int i0 = 0; i0 < rows; i0 += kBatch) {
      float in[kBatch];                              // requested together: the stores below could alias later loads
#pragma unroll
      for (int i = 0; i < kBatch; ++i) in[i] = i0 + i < rows ? load_act(a.xy, (long long)(r0 + i0 + i) * a.xy_ld + a.width + c, a.f32) : 0.f;
#pragma unroll
      for (int i = 0; i < kBatch; ++i) {
#pragma unroll
        for (int j = 0; j + 1 < kConvWin; ++j) x[j] = x[j + 1];
        x[kConvWin - 1] = in[i];
        float v = bias;
#pragma unroll
        for (int j = 0; j < kConvWin; ++j) v = fmaf(k[j], x[j], v);
        if (i0 + i < rows) store_act(a.u, u0 + (i0 + i) * ustep, v, a.f32);
      }
    }
  } else {
    for (int i = 0; i < rows; ++i) {
      float v = bias;
      for (int j = 0; j < a.taps; ++j) v = fmaf(bf(a.conv + (size_t)c * a.taps + j), conv_input(a, r0 + i - (a.taps - 1 - j), c, pos0), v);
      store_act(a.u, u0 + i * ustep, v, a.f32);
    }
  }
}

// ------------------------------------------------------------------------------------ gated linear recurrence
constexpr int kScanTokens = 64;               // tokens per CTA of the scan

// Pass 1: decay and drive of every token replace the gate pre-activations in place; decay product and end state (from zero)
// of every 64-token piece.
__global__ void __launch_bounds__(128) stack_scan_pieces_kernel(const RecurrenceArgs p) {
  griddep_wait();
  griddep_launch();
  const int c = blockIdx.y * 128 + threadIdx.x;
  if (c >= p.width) return;
  const int b = c / p.block, cb = c - b * p.block;
  const float sp = p.softplus_lam[c];
  const int r0 = blockIdx.x * kScanTokens, r1 = min(p.rows, r0 + kScanTokens);
  float* g = const_cast<float*>(p.gates) + (long long)b * 2 * p.block + cb;
  const long long gs = (long long)p.blocks * 2 * p.block, u0 = (long long)b * p.block_pad + cb, us = (long long)p.blocks * p.block_pad;
  float prod = 1.f, s = 0.f;
#pragma unroll 1
  for (int q0 = r0; q0 < r1; q0 += kBatch) {
    float zr[kBatch], zi[kBatch], u[kBatch];
#pragma unroll
    for (int i = 0; i < kBatch; ++i) {
      const int r = min(q0 + i, r1 - 1);
      zr[i] = g[r * gs];
      zi[i] = g[r * gs + p.block];
      u[i] = load_act(p.u, u0 + r * us, p.f32);
    }
#pragma unroll
    for (int i = 0; i < kBatch; ++i) {
      if (q0 + i >= r1) break;
      const float la = -p.decay * sigmoid_f(zr[i]) * sp;
      const float a = expf(la), drive = sqrtf(-expm1f(2.0f * la)) * sigmoid_f(zi[i]) * u[i];
      g[(q0 + i) * gs] = a;
      g[(q0 + i) * gs + p.block] = drive;
      prod *= a;
      s = fmaf(a, s, drive);
    }
  }
  float* o = p.agg + (size_t)blockIdx.x * 2 * p.width;
  o[c] = prod;
  o[p.width + c] = s;
}

// pass 2: state at the piece's start from the carried state and the earlier pieces, then the piece itself; the last
// piece leaves the state behind and appends the convolution history.
__global__ void __launch_bounds__(128) stack_scan_kernel(const RecurrenceArgs p) {
  griddep_wait();
  griddep_launch();
  const int c = blockIdx.y * 128 + threadIdx.x;
  const int pos0 = *p.pos0;
  const int slot = state_slot(p.tags, pos0, p.status);
  const bool last = blockIdx.x == gridDim.x - 1;
  if (slot < 0) return;
  if (c < p.width) {
    const int b = c / p.block, cb = c - b * p.block;
    float s = pos0 == 0 ? 0.f : p.state[(size_t)slot * p.width + c];
#pragma unroll 8
    for (int q = 0; q < (int)blockIdx.x; ++q) {
      const float* g = p.agg + (size_t)q * 2 * p.width;
      s = fmaf(g[c], s, g[p.width + c]);
    }
    const int r0 = blockIdx.x * kScanTokens, r1 = min(p.rows, r0 + kScanTokens);
    const float* g = p.gates + (long long)b * 2 * p.block + cb;
    const long long gs = (long long)p.blocks * 2 * p.block;
#pragma unroll 1
    for (int q0 = r0; q0 < r1; q0 += kBatch) {
      float ga[kBatch], gd[kBatch], y[kBatch];
#pragma unroll
      for (int i = 0; i < kBatch; ++i) {
        const int r = min(q0 + i, r1 - 1);
        ga[i] = g[r * gs];
        gd[i] = g[r * gs + p.block];
        y[i] = load_act(p.xy, (long long)r * p.xy_ld + c, p.f32);
      }
#pragma unroll
      for (int i = 0; i < kBatch; ++i) {
        if (q0 + i >= r1) break;
        s = fmaf(ga[i], s, gd[i]);
        store_act(p.out, (long long)(q0 + i) * p.out_ld + c, s * y[i], p.f32);
      }
    }
    if (last) {
      p.state[(size_t)(1 - slot) * p.width + c] = s;
      const int keep = min(p.taps - 1, p.rows);
      for (int j = p.rows - keep; j < p.rows; ++j)
        p.history[(long long)((pos0 + j) % p.hist_rows) * p.width + c] = load_act(p.xy, (long long)j * p.xy_ld + p.width + c, p.f32);
    }
  }
  // A CTA that starts after this store still finds `pos0` in its own slot: only the other slot's tag changes.
  if (last && blockIdx.y == 0 && threadIdx.x == 0) {
    p.tags[1 - slot] = pos0 + p.rows;
    if (pos0 == 0) p.tags[1] = -1;
  }
}

// ------------------------------------------------------------------------------------ expert rows
// Selection for chunk rows from a filled score matrix, experts limited to the best groups; one CTA per 16 rows.
__global__ void __launch_bounds__(256) stack_route_kernel(const RouterArgs a_in, const int groups, const int keep) {
  __shared__ RouterSmem sm;
  griddep_wait();
  griddep_launch();
  RouterArgs a = a_in;
  const int r0 = blockIdx.x * kRouterRows;
  a.rows = min(kRouterRows, a_in.rows - r0);
  a.scores += (size_t)r0 * a.experts;
  a.topk_ids += (size_t)r0 * a.top_k;
  a.topk_p += (size_t)r0 * a.top_k;
  router_select<true>(a, sm, true, nullptr, nullptr, nullptr, groups, keep);
}

__global__ void __launch_bounds__(128) moe_gather_kernel(const MoeGatherArgs a) {
  griddep_wait();
  griddep_launch();
  const int r = blockIdx.x, j = blockIdx.y;
  const int slot = a.slot_of[(size_t)r * a.top_k + j];
  if (!NRT_INDEX_OK(slot, a.cap, kBoundsExpert)) return;
  const uint4* src = reinterpret_cast<const uint4*>(reinterpret_cast<const char*>(a.h) + (size_t)r * a.h_ld);
  uint4* dst = reinterpret_cast<uint4*>(reinterpret_cast<char*>(a.sorted) + (size_t)slot * a.h_ld);
  for (int i = threadIdx.x; i < a.row_bytes / 16; i += 128) dst[i] = src[i];
}

}  // namespace

#define S(stream) reinterpret_cast<cudaStream_t>(stream)

extern "C" int nrt_stack_row_args_size() { return (int)sizeof(StackRowArgs); }
extern "C" int nrt_latent_prep_args_size() { return (int)sizeof(LatentPrepArgs); }
extern "C" int nrt_recurrence_args_size() { return (int)sizeof(RecurrenceArgs); }
extern "C" int nrt_moe_gather_args_size() { return (int)sizeof(MoeGatherArgs); }
extern "C" int nrt_stack_scan_tokens() { return kScanTokens; }

extern "C" int nrt_stack_rows(const void* args, void* stream) {
  StackRowArgs a;
  memcpy(&a, args, sizeof(a));
  if (a.rows < 1 || a.width < 1 || (a.y && !a.post_w) || (a.y2 && (!a.y || a.slot_of || !a.join_w || !a.join_w2))) return -3;
  const size_t smem = (size_t)a.width * 8;
  if (smem > 200 * 1024) return -7;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(stack_rows_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  return launch_pdl(stack_rows_kernel, dim3(a.rows), dim3(256), smem, S(stream), false, a);
}

extern "C" int nrt_latent_prep(const void* args, void* stream) {
  LatentPrepArgs a;
  memcpy(&a, args, sizeof(a));
  if (a.rows < 1 || a.q_rank < 1 || a.kv_rank < 1) return -3;
  return launch_pdl(latent_prep_kernel, dim3(a.rows, 2), dim3(256), 0, S(stream), false, a);
}

extern "C" int nrt_stack_conv(const void* args, void* stream) {
  RecurrenceArgs a;
  memcpy(&a, args, sizeof(a));
  if (a.rows < 1 || a.taps < 1 || a.hist_rows < 2 * (a.taps - 1) || a.hist_rows < 1 || a.width != a.blocks * a.block) return -3;
  return launch_pdl(stack_conv_kernel, dim3((a.rows + kConvRows - 1) / kConvRows, (a.width + 127) / 128), dim3(128), 0, S(stream), false, a);
}

// The recurrence over the chunk's rows: pieces, then the scan with the state hand-over.
extern "C" int nrt_stack_scan(const void* args, void* stream) {
  RecurrenceArgs a;
  memcpy(&a, args, sizeof(a));
  if (a.rows < 1 || a.width != a.blocks * a.block) return -3;
  const int pieces = (a.rows + kScanTokens - 1) / kScanTokens;
  const dim3 grid(pieces, (a.width + 127) / 128);
  int rc = 0;
  if ((rc = launch_pdl(stack_scan_pieces_kernel, grid, dim3(128), 0, S(stream), false, a))) return rc;
  return launch_pdl(stack_scan_kernel, grid, dim3(128), 0, S(stream), false, a);
}

extern "C" int nrt_stack_route(const void* args, int groups, int keep, void* stream) {
  RouterArgs a;
  memcpy(&a, args, sizeof(a));
  if (a.rows < 1 || a.experts > 256 || a.top_k > 32 || groups < 1 || groups > 32 || a.experts % groups || !a.scores || a.probs) return -3;
  return launch_pdl(stack_route_kernel, dim3((a.rows + kRouterRows - 1) / kRouterRows), dim3(256), 0, S(stream), false, a, groups, keep);
}

extern "C" int nrt_moe_gather(const void* args, void* stream) {
  MoeGatherArgs a;
  memcpy(&a, args, sizeof(a));
  if (a.rows < 1 || a.row_bytes % 16 || a.h_ld % 16) return -3;
  return launch_pdl(moe_gather_kernel, dim3(a.rows, a.top_k), dim3(128), 0, S(stream), false, a);
}
