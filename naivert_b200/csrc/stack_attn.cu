// Grouped-query attention of layer stacks around the chunk kernels of latent_attn.cu: preparation of queries, keys and values
// (norm per head, rotary positions, cache rows), the feature-major copy of the values, and the one-token step.
#include "stack.cuh"
#include "launch.hpp"

#include <string.h>

using namespace nrt;

namespace {

constexpr int kMaxHead = 512;                 // head width the kernels hold in shared memory

// One head of a token, by one warp: x[0, n) -> normed (w != null) and rotated by the angles in (cs, sn), times `scale`, in `out`
// (shared, n values).  All reads of `src` happen before the first write of `out`.
__device__ __forceinline__ void head_vector(const float* src, int n, const __nv_bfloat16* w, float eps, int half, const float* cs, const float* sn,
                                            float scale, float* out, int lane) {
  float ss = 0.f;
  for (int c = lane; c < n; c += 32) {
    const float v = __ldcg(src + c);
    out[c] = v;
    ss = fmaf(v, v, ss);
  }
  if (w) {
    const float r = 1.0f / sqrtf(lane_sum(ss) / (float)n + eps);
    for (int c = lane; c < n; c += 32) out[c] = out[c] * r * bf(w + c);
  }
  __syncwarp();
  for (int i = lane; i < half; i += 32) {
    const float u = out[i], v = out[i + half], c = cs[i], s = sn[i];
    out[i] = u * c - v * s;
    out[i + half] = v * c + u * s;
  }
  __syncwarp();
  if (scale != 1.f)
    for (int c = lane; c < n; c += 32) out[c] *= scale;
  __syncwarp();
}
__device__ __forceinline__ void angles(const GroupPrepArgs& p, int pos, float* cs, float* sn) {
  for (int i = threadIdx.x; i < p.rot_dims / 2; i += blockDim.x) sincosf((float)pos * p.freq[i], sn + i, cs + i);
}

// ------------------------------------------------------------------------------------ chunk path: preparation
// One CTA per row; a warp takes one head at a time: queries, then keys, then values.
__global__ void __launch_bounds__(256) group_prep_kernel(const GroupPrepArgs p) {
  __shared__ float buf[8][kMaxHead], cs[kMaxHead / 2], sn[kMaxHead / 2];
  griddep_wait();
  griddep_launch();
  const int r = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, half = p.rot_dims / 2;
  const int pos = *p.pos0 + r;
  if (pos < 0 || pos >= p.capacity) return;
  angles(p, pos, cs, sn);
  __syncthreads();
  const float* row = p.proj + r * p.ld;
  for (int u = warp; u < p.heads + 2 * p.kv_heads; u += 8) {
    if (u < p.heads + p.kv_heads) {
      const bool is_q = u < p.heads;
      const int h = is_q ? u : u - p.heads;
      head_vector(row + (is_q ? p.q_off : p.k_off) + h * p.dim, p.dim, is_q ? p.q_norm : p.k_norm, p.eps, half, cs, sn, is_q ? p.scale : 1.f, buf[warp], lane);
      void* dst = is_q ? p.q : p.k_cache;
      const long long at = is_q ? ((long long)r * p.heads + h) * p.dp : ((long long)pos * p.kv_heads + h) * p.dp;
      for (int c = lane; c < p.dp; c += 32) store_act(dst, at + c, c < p.dim ? buf[warp][c] : 0.f, p.f32);
      __syncwarp();
    } else {
      const int h = u - p.heads - p.kv_heads;
      for (int c = lane; c < p.vdim; c += 32) store_act(p.v_cache, ((long long)pos * p.kv_heads + h) * p.vp + c, __ldg(row + p.v_off + h * p.vdim + c), p.f32);
    }
  }
}

// dst[c][r] = src[r][c], 64 x 64 tiles, two values per access; rows beyond the last become zeros up to the tile's end
__global__ void __launch_bounds__(256) transpose_kernel(const TransposeArgs a) {
  __shared__ __nv_bfloat16 tile[64][66];
  griddep_wait();
  griddep_launch();
  const int r0 = blockIdx.x * 64, c0 = blockIdx.y * 64, tx = (threadIdx.x & 31) * 2, ty = threadIdx.x >> 5;
#pragma unroll
  for (int i = 0; i < 64; i += 8) {
    const int r = r0 + ty + i;
    uint32_t v = 0u;
    if (r < a.rows && c0 + tx < a.cols) v = __ldg(reinterpret_cast<const uint32_t*>(a.src + (long long)r * a.cols + c0 + tx));
    *reinterpret_cast<uint32_t*>(&tile[ty + i][tx]) = v;
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < 64; i += 8) {
    const int c = c0 + ty + i;
    if (c >= a.cols || r0 + tx >= a.dst_ld) continue;
    __nv_bfloat162 v;
    v.x = tile[tx][ty + i];
    v.y = tile[tx + 1][ty + i];
    *reinterpret_cast<__nv_bfloat162*>(a.dst + (long long)c * a.dst_ld + r0 + tx) = v;
  }
}

// ------------------------------------------------------------------------------------ one token
// The splits of the context of one key head are a cluster; their partial results meet through distributed shared memory.  Every CTA
// whose keys end at the token itself prepares and stores the token's key and value (equal values where there are several).
//
// Plain form (32-bit caches, wide heads): grid (splits, key heads, groups of eight query heads); eight lanes share a key, the query
// heads of the CTA are scored together; then threads own value columns.
constexpr int kHB = 8, kTile = 64, kDecThreads = 256;

__host__ __device__ inline int group_smem_floats(int dp, int vp) { return kHB * dp + kMaxHead + kTile * kHB + 3 * kHB + kHB * vp; }

template <bool F32, int VC>                    // VC value columns per thread
__global__ void __launch_bounds__(kDecThreads) group_decode_kernel(const GroupDecodeArgs a) {
  extern __shared__ __align__(16) float sh[];
  const GroupPrepArgs& p = a.p;
  float* sq = sh;                              // [8][dp]
  float* cs = sq + kHB * p.dp;
  float* sn = cs + kMaxHead / 2;
  float* sp = sn + kMaxHead / 2;               // [64][8]
  float* sm = sp + kTile * kHB;
  float* sl = sm + kHB;
  float* scorr = sl + kHB;
  float* so = scorr + kHB;                     // [8][vp]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, l = lane & 7;
  const int split = blockIdx.x, hk = blockIdx.y, group = p.heads / p.kv_heads, h0 = blockIdx.z * kHB, nh = min(kHB, group - h0);
  const int half = p.rot_dims / 2;
  griddep_wait();
  griddep_launch();
  const int pos = *reinterpret_cast<const volatile int*>(p.pos0);
  const int start = a.window > 0 ? pos / a.window * a.window : 0, n = pos + 1 - start;
  const int per = ((n + a.splits - 1) / a.splits + kTile - 1) / kTile * kTile;
  const int j_lo = min(n, split * per), j_hi = min(n, j_lo + per);
  const bool inside = pos >= 0 && pos < p.capacity;
  angles(p, pos, cs, sn);
  for (int i = tid; i < kHB * p.dp; i += kDecThreads) sq[i] = 0.f;
  for (int i = tid; i < kHB * p.vp; i += kDecThreads) so[i] = 0.f;
  if (tid < kHB) { sm[tid] = -FLT_MAX; sl[tid] = 0.f; }
  __syncthreads();
  if (inside && j_lo < j_hi) {
    if (j_hi == n) {
      // the token's own key and value (sp is free until the first tile)
      if (warp == 0) {
        head_vector(p.proj + p.k_off + hk * p.dim, p.dim, p.k_norm, p.eps, half, cs, sn, 1.f, sp, lane);
        for (int c = lane; c < p.dim; c += 32) store_act(p.k_cache, ((long long)pos * p.kv_heads + hk) * p.dp + c, sp[c], F32);
      } else if (warp == 1) {
        for (int c = lane; c < p.vdim; c += 32)
          store_act(p.v_cache, ((long long)pos * p.kv_heads + hk) * p.vp + c, __ldcg(p.proj + p.v_off + hk * p.vdim + c), F32);
      }
    }
    for (int h = warp; h < nh; h += kDecThreads / 32)
      head_vector(p.proj + p.q_off + (hk * group + h0 + h) * p.dim, p.dim, p.q_norm, p.eps, half, cs, sn, p.scale, sq + h * p.dp, lane);
    __syncthreads();
    const int pieces = p.dp / 8;
    int vc = 32;
    while (vc < p.vdim && vc < kDecThreads) vc *= 2;
    const int subs = kDecThreads / vc, sub = tid / vc, c0 = tid & (vc - 1);
    float acc[kHB][VC];
#pragma unroll
    for (int h = 0; h < kHB; ++h)
#pragma unroll
      for (int i = 0; i < VC; ++i) acc[h][i] = 0.f;
    float m = -FLT_MAX, sum = 0.f;                                       // of head `warp`
    for (int j0 = j_lo; j0 < j_hi; j0 += kTile) {
      const int live = min(kTile, j_hi - j0);
#pragma unroll
      for (int t0 = 0; t0 < kTile; t0 += kDecThreads / 8) {
        const int t = t0 + tid / 8;
        float d[kHB];
#pragma unroll
        for (int h = 0; h < kHB; ++h) d[h] = 0.f;
        if (t < live) {
          const long long at = ((long long)(start + j0 + t) * p.kv_heads + hk) * p.dp;
#pragma unroll 2
          for (int i = l; i < pieces; i += 8) {
            float4 x, y;
            if (F32) {
              const float4* k = reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p.k_cache) + at + i * 8);
              x = __ldcg(k);
              y = __ldcg(k + 1);
            } else {
              const uint4 k = __ldcg(reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(p.k_cache) + at + i * 8));
              x = make_float4(bf16_lo(k.x), bf16_hi(k.x), bf16_lo(k.y), bf16_hi(k.y));
              y = make_float4(bf16_lo(k.z), bf16_hi(k.z), bf16_lo(k.w), bf16_hi(k.w));
            }
#pragma unroll
            for (int h = 0; h < kHB; ++h) {
              const float4 q0 = *reinterpret_cast<const float4*>(sq + h * p.dp + i * 8), q1 = *reinterpret_cast<const float4*>(sq + h * p.dp + i * 8 + 4);
              d[h] = fmaf(x.x, q0.x, fmaf(x.y, q0.y, fmaf(x.z, q0.z, fmaf(x.w, q0.w, d[h]))));
              d[h] = fmaf(y.x, q1.x, fmaf(y.y, q1.y, fmaf(y.z, q1.z, fmaf(y.w, q1.w, d[h]))));
            }
          }
        }
        float mine = 0.f;
#pragma unroll
        for (int h = 0; h < kHB; ++h) {
          float v = d[h];
          v += __shfl_xor_sync(0xffffffffu, v, 1);
          v += __shfl_xor_sync(0xffffffffu, v, 2);
          v += __shfl_xor_sync(0xffffffffu, v, 4);
          if (h == l) mine = v;
        }
        sp[t * kHB + l] = mine;
      }
      __syncthreads();
      {                                                                  // softmax of head `warp`
        const float s0 = lane < live ? sp[lane * kHB + warp] : -FLT_MAX, s1 = lane + 32 < live ? sp[(lane + 32) * kHB + warp] : -FLT_MAX;
        float mt = fmaxf(s0, s1);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mt = fmaxf(mt, __shfl_xor_sync(0xffffffffu, mt, o));
        const float mn = fmaxf(m, mt), corr = expf(m - mn);
        const float p0 = lane < live ? expf(s0 - mn) : 0.f, p1 = lane + 32 < live ? expf(s1 - mn) : 0.f;
        sum = fmaf(sum, corr, lane_sum(p0 + p1));
        m = mn;
        sp[lane * kHB + warp] = p0;
        sp[(lane + 32) * kHB + warp] = p1;
        if (lane == 0) scorr[warp] = corr;
      }
      __syncthreads();
#pragma unroll
      for (int h = 0; h < kHB; ++h)
#pragma unroll
        for (int i = 0; i < VC; ++i) acc[h][i] *= scorr[h];
#pragma unroll 4
      for (int t = sub; t < live; t += subs) {
        const float4 pa = *reinterpret_cast<const float4*>(sp + t * kHB), pb = *reinterpret_cast<const float4*>(sp + t * kHB + 4);
        const long long at = ((long long)(start + j0 + t) * p.kv_heads + hk) * p.vp;
#pragma unroll
        for (int i = 0; i < VC; ++i) {
          const int c = c0 + i * kDecThreads;
          if (c < p.vdim) {
            const float v = F32 ? __ldcg(reinterpret_cast<const float*>(p.v_cache) + at + c)
                                : __bfloat162float(__ldcg(reinterpret_cast<const __nv_bfloat16*>(p.v_cache) + at + c));
            acc[0][i] = fmaf(pa.x, v, acc[0][i]);
            acc[1][i] = fmaf(pa.y, v, acc[1][i]);
            acc[2][i] = fmaf(pa.z, v, acc[2][i]);
            acc[3][i] = fmaf(pa.w, v, acc[3][i]);
            acc[4][i] = fmaf(pb.x, v, acc[4][i]);
            acc[5][i] = fmaf(pb.y, v, acc[5][i]);
            acc[6][i] = fmaf(pb.z, v, acc[6][i]);
            acc[7][i] = fmaf(pb.w, v, acc[7][i]);
          }
        }
      }
      __syncthreads();                                                   // sp is rewritten
    }
    if (lane == 0) { sm[warp] = m; sl[warp] = sum; }
    // key subsets join in a fixed order
    for (int s = 0; s < subs; ++s) {
      if (sub == s) {
#pragma unroll
        for (int h = 0; h < kHB; ++h)
#pragma unroll
          for (int i = 0; i < VC; ++i)
            if (c0 + i * kDecThreads < p.vdim) so[h * p.vp + c0 + i * kDecThreads] += acc[h][i];
      }
      __syncthreads();
    }
  }
  cluster_sync_all();
  // every CTA of the cluster finishes a share of the heads' columns
  for (int i = split * kDecThreads + tid; i < nh * p.vdim; i += a.splits * kDecThreads) {
    const int h = i / p.vdim, c = i - h * p.vdim;
    float m = -FLT_MAX, o = 0.f, sum = 0.f;
    for (int s = 0; s < a.splits; ++s) m = fmaxf(m, ld_cluster_f32(sm + h, s));
    for (int s = 0; s < a.splits; ++s) {
      const float w = expf(ld_cluster_f32(sm + h, s) - m);
      sum = fmaf(w, ld_cluster_f32(sl + h, s), sum);
      o = fmaf(w, ld_cluster_f32(so + h * p.vp + c, s), o);
    }
    a.out[(long long)(hk * group + h0 + h) * p.vp + c] = o / sum;
  }
  cluster_sync_all();                                                    // nobody leaves while its shared memory is read
}

// Tensor-core form: grid (splits, key heads, tiles of 16 or 32 query heads).  The query heads of a key head are the M side of bf16
// m16n8k16 MMAs; keys and values come 64 at a time through two to four cp.async stages, the first requested before the wait for the
// predecessor (older rows do not depend on it; the token's own row is put into its tile by hand).  tcgen05 is not used: the kernel
// streams the cache once, and most of its M = 128 rows would idle.
constexpr int kTcHead = 256;
__host__ __device__ inline int tc_pitch(int n) { return (n + 15) / 16 * 16 + 8; }              // bf16 elements; rows fall into distinct banks
__host__ __device__ inline int group_tc_smem(int dp, int vp, int ht, int stages) {
  return 2 * (ht + stages * kTile) * tc_pitch(dp) + 2 * stages * kTile * tc_pitch(vp) + 4 * ht * (kTile + 4) + 2 * ht * (kTile + 8) + 4 * 3 * ht + 4 * ht * vp +
         4 * (8 * kTcHead + kTcHead) + 2 * (dp + vp);
}

template <int MT>
__global__ void __launch_bounds__(kDecThreads, 1) group_decode_tc_kernel(const GroupDecodeArgs a, const int stages) {
  extern __shared__ __align__(16) uint8_t raw[];
  constexpr int HT = MT * 16, kSP = kTile + 4, kPP = kTile + 8, kNT = kTcHead / 64;
  const GroupPrepArgs& p = a.p;
  const int kp = tc_pitch(p.dp), vpitch = tc_pitch(p.vp), rp = (p.dp + 15) / 16 * 16;
  __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(raw);             // [HT][kp]
  __nv_bfloat16* sk = sq + HT * kp;                                      // [stages][64][kp]
  __nv_bfloat16* sv = sk + stages * kTile * kp;                          // [stages][64][vpitch]
  __nv_bfloat16* sp = sv + stages * kTile * vpitch;                           // [HT][kPP]
  float* ss = reinterpret_cast<float*>(sp + HT * kPP);                   // [HT][kSP]
  float* sm = ss + HT * kSP;
  float* sl = sm + HT;
  float* scorr = sl + HT;
  float* so = scorr + HT;                                                // [HT][vp]
  float* cs = so + HT * p.vp;
  float* sn = cs + kTcHead / 2;
  float* buf = sn + kTcHead / 2;                                         // [8][256]
  __nv_bfloat16* new_k = reinterpret_cast<__nv_bfloat16*>(buf + 8 * kTcHead);
  __nv_bfloat16* new_v = new_k + p.dp;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int split = blockIdx.x, hk = blockIdx.y, group = p.heads / p.kv_heads, h0 = blockIdx.z * HT, nh = min(HT, group - h0);
  const int half = p.rot_dims / 2;
  const int pos = *reinterpret_cast<const volatile int*>(p.pos0);
  const bool inside = pos >= 0 && pos < p.capacity;
  const int start = a.window > 0 ? pos / a.window * a.window : 0, n = inside ? pos + 1 - start : 0;
  const int per = ((n + a.splits - 1) / a.splits + kTile - 1) / kTile * kTile;
  const int j_lo = min(n, split * per), j_hi = min(n, j_lo + per);
  const bool owner = j_hi == n && j_lo < j_hi;
  {
    uint4* z = reinterpret_cast<uint4*>(raw);                            // columns beyond a head stay zero
    const int words = ((HT + stages * kTile) * kp + stages * kTile * vpitch) / 8;
    for (int i = tid; i < words; i += kDecThreads) z[i] = make_uint4(0u, 0u, 0u, 0u);
  }
  for (int i = tid; i < HT * p.vp; i += kDecThreads) so[i] = 0.f;
  for (int i = tid; i < HT; i += kDecThreads) { sm[i] = -FLT_MAX; sl[i] = scorr[i] = 0.f; }
  for (int i = tid; i < HT * kPP; i += kDecThreads) sp[i] = __float2bfloat16_rn(0.f);
  __syncthreads();
  const __nv_bfloat16* kc = reinterpret_cast<const __nv_bfloat16*>(p.k_cache) + (long long)hk * p.dp;
  const __nv_bfloat16* vc = reinterpret_cast<const __nv_bfloat16*>(p.v_cache) + (long long)hk * p.vp;
  // a thread copies one 16-byte piece of every so-many-th row
  auto rows_in = [&](int j0, __nv_bfloat16* dst, int pitch, const __nv_bfloat16* src, int width) {
    int lanes = 1;
    while (lanes < width / 8) lanes *= 2;
    const int c = tid & (lanes - 1), step = kDecThreads / lanes;
    if (c >= width / 8) return;
    const long long row_step = (long long)p.kv_heads * width;
    int t = tid / lanes;
    const __nv_bfloat16* s0 = src + (long long)(start + j0 + t) * row_step + c * 8;
    __nv_bfloat16* d = dst + t * pitch + c * 8;
#pragma unroll 4
    for (; t < kTile; t += step, s0 += step * row_step, d += step * pitch) {
      const bool in = j0 + t < j_hi && j0 + t != n - 1;                  // the token's own row is not in the cache yet
      cp16(d, in ? s0 : src, in);
    }
  };
  auto request = [&](int j0, int st) {         // the 64 rows from j0 on (none beyond the split: an empty group keeps the count)
    if (j0 < j_hi) {
      rows_in(j0, sk + st * kTile * kp, kp, kc, p.dp);
      rows_in(j0, sv + st * kTile * vpitch, vpitch, vc, p.vp);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  for (int i = 0; i + 1 < stages; ++i) request(j_lo + i * kTile, i);
  griddep_wait();
  griddep_launch();
  if (j_lo < j_hi) {
    angles(p, pos, cs, sn);
    __syncthreads();
    for (int u = warp; u < nh + (owner ? 2 : 0); u += kDecThreads / 32) {
      float* b = buf + warp * kTcHead;
      if (u < nh) {
        head_vector(p.proj + p.q_off + (hk * group + h0 + u) * p.dim, p.dim, p.q_norm, p.eps, half, cs, sn, p.scale, b, lane);
        for (int c = lane; c < p.dim; c += 32) sq[u * kp + c] = __float2bfloat16_rn(b[c]);
      } else if (u == nh) {
        head_vector(p.proj + p.k_off + hk * p.dim, p.dim, p.k_norm, p.eps, half, cs, sn, 1.f, b, lane);
        for (int c = lane; c < p.dp; c += 32) {
          const __nv_bfloat16 x = __float2bfloat16_rn(c < p.dim ? b[c] : 0.f);
          new_k[c] = x;
          reinterpret_cast<__nv_bfloat16*>(p.k_cache)[((long long)pos * p.kv_heads + hk) * p.dp + c] = x;
        }
      } else {
        for (int c = lane; c < p.vp; c += 32) {
          const __nv_bfloat16 x = __float2bfloat16_rn(c < p.vdim ? __ldcg(p.proj + p.v_off + hk * p.vdim + c) : 0.f);
          new_v[c] = x;
          reinterpret_cast<__nv_bfloat16*>(p.v_cache)[((long long)pos * p.kv_heads + hk) * p.vp + c] = x;
        }
      }
      __syncwarp();
    }
    float o[MT][kNT][4];
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int t = 0; t < kNT; ++t)
#pragma unroll
        for (int q = 0; q < 4; ++q) o[i][t][q] = 0.f;
    const int ntiles = p.vp / 8, fr = lane >> 2, fc = (lane & 3) * 2;
    const float c2 = 1.4426950408889634f;                                // scores in powers of two
    int st = 0;
    for (int j0 = j_lo; j0 < j_hi; j0 += kTile, st = st + 1 == stages ? 0 : st + 1) {
      request(j0 + (stages - 1) * kTile, st == 0 ? stages - 1 : st - 1);
      if (stages == 4) asm volatile("cp.async.wait_group 3;" ::: "memory");
      else if (stages == 3) asm volatile("cp.async.wait_group 2;" ::: "memory");
      else asm volatile("cp.async.wait_group 1;" ::: "memory");
      __syncthreads();
      if (owner && n - 1 < j0 + kTile) {                                 // the last tile: the token's own row
        for (int c = tid; c < p.dp; c += kDecThreads) sk[(st * kTile + n - 1 - j0) * kp + c] = new_k[c];
        for (int c = tid; c < p.vp; c += kDecThreads) sv[(st * kTile + n - 1 - j0) * vpitch + c] = new_v[c];
        __syncthreads();
      }
      const __nv_bfloat16* kt = sk + st * kTile * kp;
      const __nv_bfloat16* vt = sv + st * kTile * vpitch;
      // scores: warp = 8 keys, all heads
      float acc[MT][2][4];                                               // even and odd steps: two chains
#pragma unroll
      for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int q = 0; q < 8; ++q) acc[i][q >> 2][q & 3] = 0.f;
      const __nv_bfloat16* krow = kt + (warp * 8 + (lane & 7)) * kp + ((lane >> 3) & 1) * 8;
      const __nv_bfloat16* qrow = sq + (lane & 15) * kp + (lane >> 4) * 8;
#pragma unroll 2
      for (int k = 0; k < rp; k += 32) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          if (e && k + 16 >= rp) break;
          uint32_t b0, b1;
          ldsm2(b0, b1, krow + k + 16 * e);
#pragma unroll
          for (int i = 0; i < MT; ++i) {
            uint32_t af[4];
            ldsm4(af, qrow + i * 16 * kp + k + 16 * e);
            mma16816(acc[i][e], af, b0, b1);
          }
        }
      }
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        float* d = ss + (i * 16 + fr) * kSP + warp * 8 + fc;
        d[0] = (acc[i][0][0] + acc[i][1][0]) * c2;
        d[1] = (acc[i][0][1] + acc[i][1][1]) * c2;
        d[8 * kSP] = (acc[i][0][2] + acc[i][1][2]) * c2;
        d[8 * kSP + 1] = (acc[i][0][3] + acc[i][1][3]) * c2;
      }
      __syncthreads();
      const int live = j_hi - j0;
#pragma unroll
      for (int ti = 0; ti < HT / 8; ++ti) {
        const int t = warp + 8 * ti;
        if (t >= nh) break;                                              // (rows without a head stay zero)
        const float s0 = lane < live ? ss[t * kSP + lane] : -FLT_MAX, s1 = lane + 32 < live ? ss[t * kSP + lane + 32] : -FLT_MAX;
        float mt = fmaxf(s0, s1);
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) mt = fmaxf(mt, __shfl_xor_sync(0xffffffffu, mt, off));
        const float m_old = sm[t], mn = fmaxf(m_old, mt), corr = exp2_approx(m_old - mn);
        const float p0 = lane < live ? exp2_approx(s0 - mn) : 0.f, p1 = lane + 32 < live ? exp2_approx(s1 - mn) : 0.f;
        const float l = lane_sum(p0 + p1);
        sp[t * kPP + lane] = __float2bfloat16_rn(p0);
        sp[t * kPP + lane + 32] = __float2bfloat16_rn(p1);
        __syncwarp();
        if (lane == 0) { sm[t] = mn; sl[t] = sl[t] * corr + l; scorr[t] = corr; }
      }
      __syncthreads();
      // outputs: warp = every eighth group of 8 value columns
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        const float ca = scorr[i * 16 + fr], cb = scorr[i * 16 + fr + 8];
        uint32_t pf[4][4];
#pragma unroll
        for (int k = 0; k < 4; ++k) ldsm4(pf[k], sp + (i * 16 + (lane & 15)) * kPP + k * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int t = 0; t < kNT; ++t) {
          const int nt = warp + 8 * t;
          if (nt >= ntiles) continue;
          o[i][t][0] *= ca;
          o[i][t][1] *= ca;
          o[i][t][2] *= cb;
          o[i][t][3] *= cb;
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            uint32_t b0, b1;
            ldsm2t(b0, b1, vt + (k * 16 + (lane & 15)) * vpitch + nt * 8);
            mma16816(o[i][t], pf[k], b0, b1);
          }
        }
      }
      __syncthreads();                                                   // the stage and the P tile are free again
    }
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int t = 0; t < kNT; ++t) {
        const int c = (warp + 8 * t) * 8 + fc;
        if (c >= p.vp) continue;
        *reinterpret_cast<float2*>(so + (i * 16 + fr) * p.vp + c) = make_float2(o[i][t][0], o[i][t][1]);
        *reinterpret_cast<float2*>(so + (i * 16 + fr + 8) * p.vp + c) = make_float2(o[i][t][2], o[i][t][3]);
      }
  }
  cluster_sync_all();
  // every CTA of the cluster finishes a share of the heads' columns
  for (int i = split * kDecThreads + tid; i < nh * p.vdim && inside; i += a.splits * kDecThreads) {
    const int h = i / p.vdim, c = i - h * p.vdim;
    float m = -FLT_MAX, v = 0.f, sum = 0.f;
    for (int s = 0; s < a.splits; ++s) m = fmaxf(m, ld_cluster_f32(sm + h, s));
    for (int s = 0; s < a.splits; ++s) {
      const float w = exp2_approx(ld_cluster_f32(sm + h, s) - m);
      sum = fmaf(w, ld_cluster_f32(sl + h, s), sum);
      v = fmaf(w, ld_cluster_f32(so + h * p.vp + c, s), v);
    }
    a.out[(long long)(hk * group + h0 + h) * p.vp + c] = v / sum;
  }
  cluster_sync_all();                                                    // nobody leaves while its shared memory is read
}

template <int MT>
int launch_decode_tc(const GroupDecodeArgs& a, cudaStream_t stream, bool pdl) {
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(group_decode_tc_kernel<MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 225 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const int group = a.p.heads / a.p.kv_heads;
  int stages = 4;
  while (stages > 2 && group_tc_smem(a.p.dp, a.p.vp, MT * 16, stages) > 220 * 1024) --stages;
  return launch_cluster(group_decode_tc_kernel<MT>, dim3(a.splits, a.p.kv_heads, (group + MT * 16 - 1) / (MT * 16)), dim3(kDecThreads), dim3(a.splits, 1, 1),
                        group_tc_smem(a.p.dp, a.p.vp, MT * 16, stages), stream, pdl, a, stages);
}

template <bool F32, int VC>
int launch_decode(const GroupDecodeArgs& a, cudaStream_t stream, bool pdl) {
  const int smem = 4 * group_smem_floats(a.p.dp, a.p.vp);
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(group_decode_kernel<F32, VC>, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const int group = a.p.heads / a.p.kv_heads;
  return launch_cluster(group_decode_kernel<F32, VC>, dim3(a.splits, a.p.kv_heads, (group + kHB - 1) / kHB), dim3(kDecThreads), dim3(a.splits, 1, 1), smem, stream,
                        pdl, a);
}

bool prep_ok(const GroupPrepArgs& p) {
  return p.heads >= 1 && p.kv_heads >= 1 && p.heads % p.kv_heads == 0 && p.dim >= 1 && p.dim <= p.dp && p.dp <= kMaxHead && p.vdim >= 1 &&
         p.vdim <= p.vp && p.vp <= kMaxHead && p.dp % 8 == 0 && p.vp % 8 == 0 && p.rot_dims >= 0 && p.rot_dims % 2 == 0 && p.rot_dims <= p.dim &&
         (p.rot_dims == 0 || p.freq) && p.rows >= 1;
}

}  // namespace

#define S(stream) reinterpret_cast<cudaStream_t>(stream)

extern "C" int nrt_group_prep_args_size() { return (int)sizeof(GroupPrepArgs); }
extern "C" int nrt_transpose_args_size() { return (int)sizeof(TransposeArgs); }
extern "C" int nrt_group_decode_args_size() { return (int)sizeof(GroupDecodeArgs); }

extern "C" int nrt_group_prep(const void* args, void* stream) {
  GroupPrepArgs p;
  memcpy(&p, args, sizeof(p));
  if (!prep_ok(p) || !p.q) return -3;
  return launch_pdl(group_prep_kernel, dim3(p.rows), dim3(256), 0, S(stream), false, p);
}

extern "C" int nrt_transpose(const void* args, void* stream) {
  TransposeArgs a;
  memcpy(&a, args, sizeof(a));
  if (a.rows < 1 || a.cols < 1 || a.cols % 2 || a.dst_ld % 2 || a.dst_ld < a.rows) return -3;
  return launch_pdl(transpose_kernel, dim3((a.rows + 63) / 64, (a.cols + 63) / 64), dim3(256), 0, S(stream), false, a);
}

extern "C" int nrt_group_decode(const void* args, void* stream, int pdl) {
  GroupDecodeArgs a;
  memcpy(&a, args, sizeof(a));
  if (!prep_ok(a.p) || a.p.rows != 1 || a.splits < 1 || a.splits > 8 || a.window < 0) return -3;
  const bool wide = a.p.vdim > kDecThreads, p = pdl != 0;
  if (!a.p.f32 && a.p.dp <= kTcHead && a.p.vp <= kTcHead) return a.p.heads / a.p.kv_heads <= 16 ? launch_decode_tc<1>(a, S(stream), p) : launch_decode_tc<2>(a, S(stream), p);
  if (a.p.f32) return wide ? launch_decode<true, 2>(a, S(stream), p) : launch_decode<true, 1>(a, S(stream), p);
  return wide ? launch_decode<false, 2>(a, S(stream), p) : launch_decode<false, 1>(a, S(stream), p);
}
