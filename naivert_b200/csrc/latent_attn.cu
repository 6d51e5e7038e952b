// Latent attention: causal softmax attention whose keys and values are linear images of one cached latent per token.
//   chunk path   keys and values of a block of cached positions are expanded by products (stack_gemm.cu), then
//                attended by the rows of the chunk; the output gate is applied as the result is stored
//                (the same kernels serve grouped-query attention from a key / value cache: `group` heads share a key head,
//                `window` limits a query to the keys of its own chunk)
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
  const int n = min(a.kv_rows, pos + 1 - a.kv0);            // visible keys of this block: [first_key, n)
  const int first_key = max(0, (a.window > 0 ? pos / a.window * a.window : 0) - a.kv0);
  const int hk = h / a.group, kv_heads = a.heads / a.group;
  const long long kld = (long long)kv_heads * a.dim, vld = (long long)kv_heads * a.vdim;
  for (int d = lane; d < a.dim; d += 32) sq[warp][d] = load_act(a.q, ((long long)r * a.heads + h) * a.dim + d, a.f32);
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
  for (int j0 = first_key; j0 < n; j0 += 32) {
    const int j = j0 + lane;
    float s = -FLT_MAX;
    if (j < n) {
      s = 0.f;
      const long long base = (long long)j * kld + hk * a.dim;
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
      const long long base = (long long)(j0 + t) * vld + hk * a.vdim;
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
      const float g = a.gate ? sigmoid_f(a.gate[(long long)r * a.gate_ld + h * a.vdim + c]) : 1.f;
      store_act(a.out, ((long long)r * a.heads + h) * a.vdim + c, o[i] * inv * g, a.f32);
    }
  }
}

// ------------------------------------------------------------------------------------ chunk path, tensor-core form
// One CTA per (head, 128 query rows); key tiles of 64; two CTAs per SM so that one's softmax runs under the other's MMAs.
//   warp 0   TMA: Q once, then K and V tiles through two stages
//   warp 1   UMMA: S = Q K^T (TMEM), then O += P V (TMEM); the next S is issued as soon as the softmax holds the last one
//   warps 2-5  softmax, one query row per thread: S from TMEM, running maximum, exponentials, P to shared memory in the
//              128-byte-swizzled K-major layout; O is rescaled in TMEM only when the maximum has grown by more than 2^8
//              (exact: the factor is carried in the sum), then normalised, gated and stored
// V comes feature-major (its product stored it so), which makes it a K-major B operand.
constexpr int kQRows = 128, kKeys = 64;
constexpr int kTcThreads = 192;

struct TcBars {
  uint64_t q_full, k_full[2], k_empty[2], v_full[2], v_empty[2], s_full, s_empty, p_full, pv_done;
  uint32_t tmem;
};

__host__ __device__ inline int tc_chunks(int dim) { return (dim + 63) / 64; }
__host__ __device__ inline int tc_n(int vdim) { return (vdim + 15) / 16 * 16; }
__host__ __device__ inline int tc_smem(int dim, int vdim) {
  return tc_chunks(dim) * (16384 + 2 * 8192) + 2 * tc_n(vdim) * 128 + 16384 + 256;
}
__host__ __device__ inline uint32_t tc_tmem_cols(int vdim) {
  uint32_t c = 32;
  while ((int)c < kKeys + tc_n(vdim)) c *= 2;
  return c;
}

__global__ void __launch_bounds__(kTcThreads) latent_attn_tc_kernel(const __grid_constant__ CUtensorMap tmQ,
                                                                    const __grid_constant__ CUtensorMap tmK,
                                                                    const __grid_constant__ CUtensorMap tmV, const LatentAttnArgs a) {
  extern __shared__ __align__(1024) uint8_t smem[];
  const int chunks = tc_chunks(a.dim), N = tc_n(a.vdim);
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + chunks * 16384;
  uint8_t* sV = sK + 2 * chunks * 8192;
  uint8_t* sP = sV + 2 * N * 128;
  TcBars* bar = reinterpret_cast<TcBars*>(sP + 16384);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // query tiles of one head run side by side (they share its keys in L2), the longest first
  const int h = blockIdx.y, r0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * kQRows;
  const uint32_t cols = tc_tmem_cols(a.vdim);
  if ((smem_u32(smem) & 1023u) != 0u) {                    // the swizzle pattern counts from a 1024-byte boundary
    if (threadIdx.x == 0) report(a.status, kSiteGrid | 0x10);
    return;
  }
  if (threadIdx.x == 0) {
    mbar_init(&bar->q_full, 1);
    for (int i = 0; i < 2; ++i) { mbar_init(&bar->k_full[i], 1); mbar_init(&bar->k_empty[i], 1); mbar_init(&bar->v_full[i], 1); mbar_init(&bar->v_empty[i], 1); }
    mbar_init(&bar->s_full, 1);
    mbar_init(&bar->s_empty, 128);
    mbar_init(&bar->p_full, 128);
    mbar_init(&bar->pv_done, 1);
    mbar_fence_init();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
  }
  if (warp == 1) { tmem_alloc(&bar->tmem, cols); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  griddep_wait();
  griddep_launch();
  const uint32_t tS = bar->tmem, tO = bar->tmem + kKeys;
  const int pos0 = *a.pos0;
  const int last_row = min(r0 + kQRows, a.rows) - 1;
  const int seen = min(a.kv_rows, pos0 + last_row + 1 - a.kv0);
  // tiles of keys that no row of this CTA sees (earlier chunks of the mask) are left out
  const int tile0 = max(0, (a.window > 0 ? (pos0 + r0) / a.window * a.window : 0) - a.kv0) / kKeys;
  const int tiles = seen > tile0 * kKeys ? (seen + kKeys - 1) / kKeys - tile0 : 0;
  const int hk = h / a.group;

  if (warp == 0) {
    if (elect_one() && tiles > 0) {
      mbar_expect_tx(&bar->q_full, chunks * 16384);
      for (int c = 0; c < chunks; ++c) tma_load_3d(sQ + c * 16384, &tmQ, &bar->q_full, c * 64, h, r0);
      for (int j = 0; j < tiles; ++j) {
        const int st = j & 1;
        const uint32_t ph = ((j >> 1) & 1) ^ 1;
        if (j >= 2 && !mbar_wait(&bar->k_empty[st], ph, a.status, kSiteStageEmpty | st)) break;
        mbar_expect_tx(&bar->k_full[st], chunks * 8192);
        for (int c = 0; c < chunks; ++c) tma_load_3d(sK + (st * chunks + c) * 8192, &tmK, &bar->k_full[st], c * 64, hk, a.k_row0 + (tile0 + j) * kKeys);
        if (j >= 2 && !mbar_wait(&bar->v_empty[st], ph, a.status, kSiteStageEmpty | 8 | st)) break;
        mbar_expect_tx(&bar->v_full[st], N * 128);
        tma_load_2d(sV + st * N * 128, &tmV, &bar->v_full[st], (tile0 + j) * kKeys, hk * a.vdim);
      }
    }
  } else if (warp == 1) {
    if (elect_one() && tiles > 0) {
      const uint32_t id_s = umma_idesc(1u, kQRows, kKeys), id_o = umma_idesc(1u, kQRows, N);
      bool ok = mbar_wait(&bar->q_full, 0, a.status, kSiteTmaFull | 0x10);
      auto scores = [&](int j) {
        const int st = j & 1;
        if (!mbar_wait(&bar->k_full[st], (j >> 1) & 1, a.status, kSiteTmaFull | st)) return false;
        tc_fence_after();
        for (int c = 0; c < chunks; ++c) {
          const uint64_t dq = umma_desc_sw128(smem_u32(sQ + c * 16384)), dk = umma_desc_sw128(smem_u32(sK + (st * chunks + c) * 8192));
#pragma unroll
          for (int q = 0; q < 4; ++q) umma_bf16(tS, dq + 2 * q, dk + 2 * q, id_s, c > 0 || q > 0);
        }
        umma_commit(&bar->k_empty[st]);
        umma_commit(&bar->s_full);
        return true;
      };
      ok = ok && scores(0);
      for (int j = 0; j < tiles && ok; ++j) {
        if (j + 1 < tiles) {
          ok = mbar_wait(&bar->s_empty, j & 1, a.status, kSiteAccEmpty) && scores(j + 1);
          if (!ok) break;
        }
        const int st = j & 1;
        ok = mbar_wait(&bar->p_full, j & 1, a.status, kSiteAccEmpty | 1) && mbar_wait(&bar->v_full[st], (j >> 1) & 1, a.status, kSiteTmaFull | 8 | st);
        if (!ok) break;
        tc_fence_after();
        const uint64_t dp = umma_desc_sw128(smem_u32(sP)), dv = umma_desc_sw128(smem_u32(sV + st * N * 128));
#pragma unroll
        for (int q = 0; q < 4; ++q) umma_bf16(tO, dp + 2 * q, dv + 2 * q, id_o, !a.first || j > 0 || q > 0);
        umma_commit(&bar->v_empty[st]);
        umma_commit(&bar->pv_done);
      }
    }
  } else {
    const int quad = warp & 3, row = quad * 32 + lane, r = r0 + row;
    const uint32_t lane_off = uint32_t(quad * 32) << 16;
    const bool live = r < a.rows;
    const int vis = min(a.kv_rows, pos0 + r + 1 - a.kv0);              // visible keys of this row in the block: [low, vis)
    const int low = a.window > 0 ? (pos0 + r) / a.window * a.window - a.kv0 : 0;
    const float c2 = a.scale * 1.4426950408889634f;                    // scores in powers of two
    float* st_row = a.state ? a.state + ((size_t)min(r, a.rows - 1) * a.heads + h) * (a.vdim + 2) : nullptr;
    float m = -INFINITY, l = 0.f;                                      // m in scaled (base 2) units
    if (!a.first) {
      m = st_row[0];
      l = st_row[1];
      if (tiles > 0) {
        for (int c = 0; c < N; c += 16) {
          uint32_t v[16];
#pragma unroll
          for (int i = 0; i < 16; ++i) v[i] = c + i < a.vdim ? __float_as_uint(st_row[2 + c + i]) : 0u;
          __syncwarp();
          tmem_st16(tO + lane_off + c, v);
        }
        tmem_st_wait();
      }
    }
    bool ok = true;
    for (int j = 0; j < tiles; ++j) {
      ok = __all_sync(0xffffffffu, mbar_wait(&bar->s_full, j & 1, a.status, kSiteAccFull));
      if (!ok) break;
      tc_fence_after();
      uint32_t s[kKeys];
#pragma unroll
      for (int q = 0; q < kKeys / 16; ++q) tmem_ld16_nowait(tS + lane_off + 16 * q, s + 16 * q);
      tmem_ld_wait();
      tc_fence_before();
      mbar_arrive(&bar->s_empty);
      const int k0 = (tile0 + j) * kKeys;
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};      // four chains: the row's 64 values are one thread's
      if (k0 + kKeys <= vis && k0 >= low) {
#pragma unroll
        for (int i = 0; i < kKeys; ++i) mx4[i & 3] = fmaxf(mx4[i & 3], __uint_as_float(s[i]));
      } else {
#pragma unroll
        for (int i = 0; i < kKeys; ++i) {
          if (k0 + i >= vis || k0 + i < low) s[i] = 0xff800000u;
          mx4[i & 3] = fmaxf(mx4[i & 3], __uint_as_float(s[i]));
        }
      }
      float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      mx *= c2;                                                        // scale > 0 keeps the order
      float corr = 1.f;
      bool grow = false;
      if (m == -INFINITY) m = mx;
      else if (mx > m + 8.f) { corr = exp2_approx(m - mx); m = mx; grow = true; }
      const float base = m == -INFINITY ? 0.f : m;
      float sum4[4] = {0.f, 0.f, 0.f, 0.f};
      uint32_t pk[kKeys / 2];
#pragma unroll
      for (int i = 0; i < kKeys; i += 2) {
        const float p0 = exp2_approx(fmaf(__uint_as_float(s[i]), c2, -base)), p1 = exp2_approx(fmaf(__uint_as_float(s[i + 1]), c2, -base));
        sum4[(i >> 1) & 3] += p0 + p1;
        pk[i / 2] = pack_bf16x2(p0, p1);
      }
      l = fmaf(l, corr, (sum4[0] + sum4[1]) + (sum4[2] + sum4[3]));
      if (j > 0) ok = __all_sync(0xffffffffu, mbar_wait(&bar->pv_done, (j - 1) & 1, a.status, kSiteAccFull | 1));
      if (!ok) break;
      if ((j > 0 || !a.first) && __any_sync(0xffffffffu, grow)) {
        tc_fence_after();
        for (int c = 0; c < N; c += 16) {
          uint32_t v[16];
          tmem_ld16_nowait(tO + lane_off + c, v);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 16; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * corr);
          tmem_st16(tO + lane_off + c, v);
        }
        tmem_st_wait();
      }
      uint4* dst = reinterpret_cast<uint4*>(sP + row * 128);
#pragma unroll
      for (int q = 0; q < 8; ++q) dst[q ^ (row & 7)] = make_uint4(pk[4 * q], pk[4 * q + 1], pk[4 * q + 2], pk[4 * q + 3]);
      fence_proxy_async_smem();
      tc_fence_before();
      mbar_arrive(&bar->p_full);
    }
    if (ok && tiles > 0) ok = __all_sync(0xffffffffu, mbar_wait(&bar->pv_done, (tiles - 1) & 1, a.status, kSiteAccFull | 1));
    if (ok) {
      tc_fence_after();
      const float inv = 1.0f / l;
      const bool gate_vec = ((reinterpret_cast<uintptr_t>(a.gate) & 15) | (a.gate_ld & 3)) == 0;
      if (!a.last && live) { st_row[0] = m; st_row[1] = l; }
      for (int c = 0; c < N; c += 16) {
        uint32_t v[16];
        if (tiles > 0) {
          __syncwarp();
          tmem_ld16_nowait(tO + lane_off + c, v);
          tmem_ld_wait();
        } else {
#pragma unroll
          for (int i = 0; i < 16; ++i) v[i] = c + i < a.vdim ? __float_as_uint(st_row[2 + c + i]) : 0u;
        }
        if (live) {
          const float* g = a.gate ? a.gate + (long long)r * a.gate_ld + (long long)h * a.vdim + c : nullptr;
          __nv_bfloat16* o = reinterpret_cast<__nv_bfloat16*>(a.out) + ((long long)r * a.heads + h) * a.vdim + c;
#pragma unroll
          for (int q = 0; q < 2; ++q) {
            if (c + 8 * q >= a.vdim) continue;                         // vdim is a multiple of 8
            if (!a.last) {
#pragma unroll
              for (int i = 0; i < 8; ++i) st_row[2 + c + 8 * q + i] = __uint_as_float(v[8 * q + i]);
            } else {
              float x[8];
              if (!a.gate) {
              } else if (gate_vec) {
                const float4 g0 = *reinterpret_cast<const float4*>(g + 8 * q), g1 = *reinterpret_cast<const float4*>(g + 8 * q + 4);
                x[0] = g0.x; x[1] = g0.y; x[2] = g0.z; x[3] = g0.w;
                x[4] = g1.x; x[5] = g1.y; x[6] = g1.z; x[7] = g1.w;
              } else {
#pragma unroll
                for (int i = 0; i < 8; ++i) x[i] = g[8 * q + i];
              }
#pragma unroll
              for (int i = 0; i < 8; ++i) x[i] = __uint_as_float(v[8 * q + i]) * inv * (a.gate ? sigmoid_f(x[i]) : 1.f);
              *reinterpret_cast<uint4*>(o + 8 * q) =
                  make_uint4(pack_bf16x2(x[0], x[1]), pack_bf16x2(x[2], x[3]), pack_bf16x2(x[4], x[5]), pack_bf16x2(x[6], x[7]));
            }
          }
        }
      }
    }
  }
  drain_on_error(a.status);
  tc_fence_before();
  __syncthreads();
  if (warp == 1) { tc_fence_after(); tmem_dealloc(bar->tmem, cols); }
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
  const int per = latent_split_rows(n, a.splits);
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
  float* out = a.part + ((size_t)sp_i * a.heads + h) * latent_part_row(a.rank);
  if (threadIdx.x == 0) { out[0] = m; out[1] = l; }
  for (int c = threadIdx.x; c < a.rank; c += 256) out[4 + c] = o[c];
}

// ------------------------------------------------------------------------------------ one-token step, tensor-core form
// grid (head tiles, splits).  Up to 32 heads of a CTA share every cached latent: the heads are the M side of bf16 m16n8k16
// MMAs, the latents (64 per tile, two cp.async stages) serve as keys and, through ldmatrix.trans, as values.  tcgen05 is not
// used: the kernel streams the cache once, and with at most 64 or so live query rows half of its M = 128 would idle.
constexpr int kMaxDecRank = 512;
__host__ __device__ inline int dec_pitch(int rank) { return (rank + 15) / 16 * 16 + 8; }        // bf16 elements; rows fall into distinct banks
__host__ __device__ inline int dec_smem(int rank, int mt) {
  return (mt * 16 + 2 * kDecTile) * dec_pitch(rank) * 2 + mt * 16 * (kDecTile + 4) * 4 + mt * 16 * (kDecTile + 8) * 2 + mt * 16 * 12;
}

template <int MT>
__global__ void __launch_bounds__(256, 1) latent_decode_tc_kernel(const LatentDecodeArgs a) {
  extern __shared__ uint4 dyn[];
  constexpr int HT = MT * 16, kSP = kDecTile + 4, kPP = kDecTile + 8, kNT = kMaxDecRank / 64;   // n8 tiles per warp
  const int rp = (a.rank + 15) / 16 * 16, pitch = dec_pitch(a.rank);
  __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(dyn);
  __nv_bfloat16* sc = sq + HT * pitch;
  float* ss = reinterpret_cast<float*>(sc + 2 * kDecTile * pitch);
  __nv_bfloat16* sp = reinterpret_cast<__nv_bfloat16*>(ss + HT * kSP);
  float* sm = reinterpret_cast<float*>(sp + HT * kPP);
  float* sl = sm + HT;
  float* scorr = sl + HT;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h0 = blockIdx.x * HT;
  // The position and the cache rows (the newest was appended two launches back) do not depend on the predecessor: the first
  // tile is requested before the wait for it.
  const int n = *reinterpret_cast<const volatile int*>(a.pos0) + 1;
  const int per = latent_split_rows(n, a.splits);
  const int j_lo = min(n, (int)blockIdx.y * per), j_hi = min(n, j_lo + per);
  const __nv_bfloat16* cache = reinterpret_cast<const __nv_bfloat16*>(a.cache);
  const int pieces = rp / 8, t_first = tid / pieces, c_first = tid - t_first * pieces, t_step = 256 / pieces, c_step = 256 - t_step * pieces;
  auto request = [&](int j0, int stage) {
    int t = t_first, c = c_first;                     // piece (t, c) of the tile; steps of 256 pieces without divisions
    while (t < kDecTile) {
      const bool in = j0 + t < j_hi;
      cp16(sc + (stage * kDecTile + t) * pitch + c * 8, cache + (long long)(in ? j0 + t : j_lo) * a.cache_ld + c * 8, in);
      c += c_step;
      t += t_step;
      if (c >= pieces) { c -= pieces; ++t; }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (j_lo < j_hi) request(j_lo, 0);
  griddep_wait();
  griddep_launch();
  if (j_lo >= j_hi) return;                           // an unused split: nobody reads its partial
  if (a.rank % 4 == 0) {
#pragma unroll 4
    for (int i = tid; i < HT * rp / 4; i += 256) {
      const int t = i / (rp / 4), c = (i - t * (rp / 4)) * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (h0 + t < a.heads && c < a.rank) v = __ldcg(reinterpret_cast<const float4*>(a.q + (size_t)(h0 + t) * a.rank + c));
      *reinterpret_cast<uint2*>(sq + t * pitch + c) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
    }
  } else
  for (int i = tid; i < HT * rp; i += 256) {
    const int t = i / rp, c = i - t * rp;
    const float v = h0 + t < a.heads && c < a.rank ? __ldcg(a.q + (size_t)(h0 + t) * a.rank + c) : 0.f;
    sq[t * pitch + c] = __float2bfloat16_rn(v);
  }
  for (int i = tid; i < HT; i += 256) { sm[i] = -FLT_MAX; sl[i] = 0.f; }
  float o[MT][kNT][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int t = 0; t < kNT; ++t)
#pragma unroll
      for (int q = 0; q < 4; ++q) o[i][t][q] = 0.f;
  const int ntiles = rp / 8;
  const float c2 = a.scale * 1.4426950408889634f;     // scores in powers of two
  int stage = 0;
  for (int j0 = j_lo; j0 < j_hi; j0 += kDecTile, stage ^= 1) {
    if (j0 + kDecTile < j_hi) {
      request(j0 + kDecTile, stage ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const __nv_bfloat16* kc = sc + stage * kDecTile * pitch;
    // scores: warp = 8 keys, all heads
    float acc[MT][4];
#pragma unroll
    for (int i = 0; i < MT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll 4
    for (int k = 0; k < rp; k += 16) {
      uint32_t b0, b1;
      ldsm2(b0, b1, kc + (warp * 8 + (lane & 7)) * pitch + k + ((lane >> 3) & 1) * 8);
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        uint32_t af[4];
        ldsm4(af, sq + (i * 16 + (lane & 15)) * pitch + k + (lane >> 4) * 8);
        mma16816(acc[i], af, b0, b1);
      }
    }
    const int fr = lane >> 2, fc = (lane & 3) * 2;
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      float* d = ss + (i * 16 + fr) * kSP + warp * 8 + fc;
      d[0] = acc[i][0] * c2;
      d[1] = acc[i][1] * c2;
      d[8 * kSP] = acc[i][2] * c2;
      d[8 * kSP + 1] = acc[i][3] * c2;
    }
    __syncthreads();
    const int live = j_hi - j0;
#pragma unroll
    for (int ti = 0; ti < HT / 8; ++ti) {
      const int t = warp + 8 * ti;
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
    // latent outputs: warp = every eighth group of 8 columns
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
          ldsm2t(b0, b1, kc + (k * 16 + (lane & 15)) * pitch + nt * 8);
          mma16816(o[i][t], pf[k], b0, b1);
        }
      }
    }
    __syncthreads();                                 // the stage and the P tile are free again
  }
  const int fr = lane >> 2, fc = (lane & 3) * 2;
  __syncthreads();
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int t = i * 16 + fr + 8 * half;
      if (h0 + t >= a.heads) continue;
      float* out = a.part + ((size_t)blockIdx.y * a.heads + h0 + t) * latent_part_row(a.rank);
      if (warp == 0 && (lane & 3) == 0) { out[0] = sm[t] * 0.6931471805599453f; out[1] = sl[t]; }     // maximum in natural units
#pragma unroll
      for (int q = 0; q < kNT; ++q) {
        const int c = (warp + 8 * q) * 8 + fc;
        if (c < a.rank) out[4 + c] = o[i][q][2 * half];
        if (c + 1 < a.rank) out[4 + c + 1] = o[i][q][2 * half + 1];
      }
    }
}

template <int MT>
int launch_decode_tc(const LatentDecodeArgs& a, cudaStream_t stream, bool pdl) {
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(latent_decode_tc_kernel<MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  return launch_pdl(latent_decode_tc_kernel<MT>, dim3((a.heads + MT * 16 - 1) / (MT * 16), a.splits), dim3(256), dec_smem(a.rank, MT), stream, pdl, a);
}

}  // namespace

extern "C" int nrt_latent_attn_args_size() { return (int)sizeof(LatentAttnArgs); }
extern "C" int nrt_latent_decode_args_size() { return (int)sizeof(LatentDecodeArgs); }

extern "C" int nrt_latent_attn_rows(const void* args, void* stream) {
  LatentAttnArgs a;
  memcpy(&a, args, sizeof(a));
  if (a.rows < 1 || a.group < 1 || a.heads % a.group || a.window < 0 || a.dim > 512 || a.vdim > 512 || ((!a.first || !a.last) && !a.state)) return -3;
  return launch_pdl(latent_attn_rows_kernel, dim3((a.rows * a.heads + 3) / 4), dim3(128), 0, reinterpret_cast<cudaStream_t>(stream), false, a);
}

// bf16; a.dim and a.vdim multiples of 8 up to 256.  tmQ / tmK: (dim, heads, rows) boxes of 64 x 1 x 128 / 64; tmV: feature-major
// (keys, heads * vdim), box 64 x pad16(vdim).
extern "C" int nrt_latent_attn_tc(const void* tmQ, const void* tmK, const void* tmV, const void* args, void* stream) {
  CUtensorMap q, k, v;
  memcpy(&q, tmQ, sizeof(q));
  memcpy(&k, tmK, sizeof(k));
  memcpy(&v, tmV, sizeof(v));
  LatentAttnArgs a;
  memcpy(&a, args, sizeof(a));
  if (a.rows < 1 || a.group < 1 || a.heads % a.group || a.window < 0 || a.f32 || a.dim > 256 || a.vdim > 256 || a.dim % 8 || a.vdim % 8 || !(a.scale > 0.f) || ((!a.first || !a.last) && !a.state)) return -3;
  const int smem = tc_smem(a.dim, a.vdim);
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(latent_attn_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  return launch_pdl(latent_attn_tc_kernel, dim3((a.rows + kQRows - 1) / kQRows, a.heads), dim3(kTcThreads), smem,
                    reinterpret_cast<cudaStream_t>(stream), false, q, k, v, a);
}

extern "C" int nrt_latent_decode(const void* args, void* stream, int pdl) {
  LatentDecodeArgs a;
  memcpy(&a, args, sizeof(a));
  if (!a.f32 && a.rank >= 1 && a.rank <= kMaxDecRank && a.splits >= 1 && a.splits <= kMaxSplits && a.cache_ld >= (a.rank + 15) / 16 * 16) {
    cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
    if (a.heads <= 16) return launch_decode_tc<1>(a, s, pdl != 0);
    return launch_decode_tc<2>(a, s, pdl != 0);
  }
  const size_t smem = (size_t)a.rank * 8;
  if (a.rank < 1 || a.splits < 1 || a.splits > kMaxSplits || smem > 48 * 1024) return -3;
  return launch_pdl(latent_decode_kernel, dim3(a.heads, a.splits), dim3(256), smem, reinterpret_cast<cudaStream_t>(stream), pdl != 0, a);
}
