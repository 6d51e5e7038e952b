// Latent attention: causal softmax attention whose keys and values are linear images of one cached latent per token.
//   chunk path   keys and values of a block of cached positions are expanded by products (stack_gemm.cu), then
//                attended by the rows of the chunk; the output gate is applied as the result is stored
//   one-token    the query is taken into the latent space instead, and the cached latents serve as keys and values
//                of all heads at once (kernels below: split over the context, merged by the next product)
#include "stack.cuh"
#include "launch.hpp"

#include <string.h>

using namespace nrt;

namespace {

// ------------------------------------------------------------------------------------ chunk path, plain form
// One warp per (row, head); keys 32 at a time.  Used by the float form; also carries state over key blocks.
__global__ void __launch_bounds__(128) latent_attn_rows_kernel(const LatentAttnArgs a) {
  __shared__ float sq[4][512];
  griddep_wait();
  griddep_launch();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int unit = blockIdx.x * 4 + warp;
  if (unit >= a.rows * a.heads) return;
  const int r = unit / a.heads, h = unit % a.heads;
  const int pos = *a.pos0 + r;
  const int n = min(a.kv_rows, pos + 1 - a.kv0);            // visible keys of this block
  const long long kld = (long long)a.heads * a.dim, vld = (long long)a.heads * a.vdim;
  for (int d = lane; d < a.dim; d += 32) sq[warp][d] = load_act(a.q, (long long)r * kld + h * a.dim + d, a.f32);
  __syncwarp();
  float o[16];
#pragma unroll
  for (int i = 0; i < 16; ++i) o[i] = 0.f;
  float m = -FLT_MAX, l = 0.f;
  float* st = a.state ? a.state + ((size_t)r * a.heads + h) * (a.vdim + 2) : nullptr;
  if (!a.first) {
    m = st[0];
    l = st[1];
#pragma unroll
    for (int i = 0; i < 16; ++i)
      if (lane + 32 * i < a.vdim) o[i] = st[2 + lane + 32 * i];
  }
  for (int j0 = 0; j0 < n; j0 += 32) {
    const int j = j0 + lane;
    float s = -FLT_MAX;
    if (j < n) {
      s = 0.f;
      const long long base = (long long)j * kld + h * a.dim;
      for (int d = 0; d < a.dim; ++d) s = fmaf(sq[warp][d], load_act(a.k, base + d, a.f32), s);
      s *= a.scale;
    }
    float mt = s;
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) mt = fmaxf(mt, __shfl_xor_sync(0xffffffffu, mt, off));
    const float mn = fmaxf(m, mt), corr = expf(m - mn);
    const float p = j < n ? expf(s - mn) : 0.f;
    l = l * corr + lane_sum(p);
    m = mn;
#pragma unroll
    for (int i = 0; i < 16; ++i) o[i] *= corr;
    const int live = min(32, n - j0);
    for (int t = 0; t < live; ++t) {
      const float pt = __shfl_sync(0xffffffffu, p, t);
      const long long base = (long long)(j0 + t) * vld + h * a.vdim;
#pragma unroll
      for (int i = 0; i < 16; ++i)
        if (lane + 32 * i < a.vdim) o[i] = fmaf(pt, load_act(a.v, base + lane + 32 * i, a.f32), o[i]);
    }
  }
  if (!a.last) {
    if (lane == 0) { st[0] = m; st[1] = l; }
#pragma unroll
    for (int i = 0; i < 16; ++i)
      if (lane + 32 * i < a.vdim) st[2 + lane + 32 * i] = o[i];
    return;
  }
  const float inv = 1.0f / l;
#pragma unroll
  for (int i = 0; i < 16; ++i) {
    const int c = lane + 32 * i;
    if (c < a.vdim) {
      const float g = sigmoid_f(a.gate[(long long)r * a.gate_ld + h * a.vdim + c]);
      store_act(a.out, (long long)r * vld + h * a.vdim + c, o[i] * inv * g, a.f32);
    }
  }
}

// ------------------------------------------------------------------------------------ one-token step, plain form
// grid (heads, splits), 256 threads; the split's keys 64 at a time.
constexpr int kDecTile = 64;
__global__ void __launch_bounds__(256) latent_decode_kernel(const LatentDecodeArgs a) {
  extern __shared__ float sh[];                 // [rank] query, [rank] output
  __shared__ float sp[kDecTile], stat[2];
  griddep_wait();
  griddep_launch();
  const int h = blockIdx.x, sp_i = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n = *a.pos0 + 1;
  const int per = ((n + a.splits - 1) / a.splits + kDecTile - 1) / kDecTile * kDecTile;
  const int j_lo = min(n, sp_i * per), j_hi = min(n, j_lo + per);
  float* q = sh;
  float* o = sh + a.rank;
  for (int c = threadIdx.x; c < a.rank; c += 256) { q[c] = a.q[(size_t)h * a.rank + c]; o[c] = 0.f; }
  float m = -FLT_MAX, l = 0.f;
  __syncthreads();
  for (int j0 = j_lo; j0 < j_hi; j0 += kDecTile) {
    const int live = min(kDecTile, j_hi - j0);
    for (int t = warp; t < live; t += 8) {
      float s = 0.f;
      for (int c = lane; c < a.rank; c += 32) s = fmaf(q[c], load_act(a.cache, (long long)(j0 + t) * a.cache_ld + c, a.f32), s);
      s = lane_sum(s);
      if (lane == 0) sp[t] = s * a.scale;
    }
    __syncthreads();
    if (warp == 0) {
      const float s0 = lane < live ? sp[lane] : -FLT_MAX, s1 = lane + 32 < live ? sp[lane + 32] : -FLT_MAX;
      float mt = fmaxf(s0, s1);
#pragma unroll
      for (int off = 16; off > 0; off >>= 1) mt = fmaxf(mt, __shfl_xor_sync(0xffffffffu, mt, off));
      const float mn = fmaxf(m, mt);
      const float p0 = lane < live ? expf(s0 - mn) : 0.f, p1 = lane + 32 < live ? expf(s1 - mn) : 0.f;
      sp[lane] = p0;
      sp[lane + 32] = p1;
      const float corr = expf(m - mn);
      l = l * corr + lane_sum(p0 + p1);
      m = mn;
      if (lane == 0) stat[0] = corr;
    }
    __syncthreads();
    const float corr = stat[0];
    for (int c = threadIdx.x; c < a.rank; c += 256) {
      float acc = o[c] * corr;
      for (int t = 0; t < live; ++t) acc = fmaf(sp[t], load_act(a.cache, (long long)(j0 + t) * a.cache_ld + c, a.f32), acc);
      o[c] = acc;
    }
    __syncthreads();
  }
  float* out = a.part + ((size_t)sp_i * a.heads + h) * (a.rank + 2);
  if (threadIdx.x == 0) { out[0] = m; out[1] = l; }
  for (int c = threadIdx.x; c < a.rank; c += 256) out[2 + c] = o[c];
}

}  // namespace

extern "C" int nrt_latent_attn_args_size() { return (int)sizeof(LatentAttnArgs); }
extern "C" int nrt_latent_decode_args_size() { return (int)sizeof(LatentDecodeArgs); }

extern "C" int nrt_latent_attn_rows(const void* args, void* stream) {
  LatentAttnArgs a;
  memcpy(&a, args, sizeof(a));
  if (a.rows < 1 || a.dim > 512 || a.vdim > 512 || ((!a.first || !a.last) && !a.state)) return -3;
  return launch_pdl(latent_attn_rows_kernel, dim3((a.rows * a.heads + 3) / 4), dim3(128), 0, reinterpret_cast<cudaStream_t>(stream), false, a);
}

extern "C" int nrt_latent_decode(const void* args, void* stream, int pdl) {
  LatentDecodeArgs a;
  memcpy(&a, args, sizeof(a));
  const size_t smem = (size_t)a.rank * 8;
  if (a.rank < 1 || a.splits < 1 || smem > 48 * 1024) return -3;
  return launch_pdl(latent_decode_kernel, dim3(a.heads, a.splits), dim3(256), smem, reinterpret_cast<cudaStream_t>(stream), pdl != 0, a);
}
