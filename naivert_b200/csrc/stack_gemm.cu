// Token-chunk products of layer stacks.
//
// Tensor-core form (bf16): features are the M = 128 side of tcgen05.mma (weights = A operand), token rows the N side
// (64, 128 or 256 per tile), both staged by TMA with 128-byte swizzle.  Persistent CTAs walk the (feature tile, item)
// list; two accumulators in TMEM let the products of the next tile run under the stores of the previous one.
//   warp 0    TMA producer        warp 1    UMMA issuer (and TMEM owner)
//   warps 2-9 epilogue: thread = feature x one half of the token columns
// An item is a row tile of one weight group (plain form: zcount groups, each reading its own columns of the token
// operand - heads or blocks with private weights) or a row segment of a routed expert (item form).  Sizes need no
// padding: the tensor maps carry the true extents and TMA fills the edges of a tile with zeros.
//
// Float form (`nrt_stack_gemm_f32`): the same products and epilogues on the CUDA cores in fp32.
#include "stack.cuh"
#include "launch.hpp"

#include <string.h>

using namespace nrt;

namespace {

constexpr int kFeat = 128;                    // features per tile
constexpr int kKStep = 64;                    // inner elements per stage (128 bytes of bf16)
constexpr int kATile = kFeat * 128;           // bytes
constexpr int kThreads = 320;

template <int NTOK, bool DUAL>
struct Cfg {
  static constexpr int kStage = (DUAL ? 2 : 1) * kATile + NTOK * 128;
  static constexpr int kStages = (200 * 1024) / kStage > 8 ? 8 : (200 * 1024) / kStage;
  static constexpr int kAccCols = (DUAL ? 2 : 1) * NTOK;
  static constexpr int kTmem = 2 * kAccCols;                     // two tiles in flight
  static constexpr int kSmem = kStages * kStage + 1024 + 512;
};
static_assert(Cfg<256, false>::kTmem == 512 && Cfg<128, true>::kTmem == 512 && Cfg<64, false>::kTmem == 128, "TMEM columns");

struct Tail {
  uint64_t full[8], empty[8], acc_full[2], acc_empty[2];
  uint32_t tmem;
};

struct Item { int z, row0; bool live; };

__device__ __forceinline__ Item item_of(const StackGemmArgs& p, int item, int row_tiles, int ntok, int na) {
  Item it;
  if (p.n_items) {
    it.live = item < na;
    it.z = it.live ? p.item_z[item] : 0;
    it.row0 = it.live ? p.item_row[item] : 0;
  } else {
    it.live = true;
    it.z = item / row_tiles;
    it.row0 = (item % row_tiles) * ntok;
  }
  return it;
}

template <int EPI>
constexpr bool epi_has_bias() { return EPI == kSEpiBias || EPI == kSEpiDecaySoft || EPI == kSEpiDecayExp; }

template <int EPI>
__device__ __forceinline__ float epi_value(const StackGemmArgs& p, float a0, float a1, int n, float bias, float rate) {
  if (EPI == kSEpiBias) {
    const float v = a0 + bias;
    return n < p.act_cols ? gelu_tanh_f(v) : v;
  }
  if (EPI == kSEpiClampedGlu) return clamped_glu(a0, a1, p.limit, p.alpha);
  if (EPI == kSEpiSiluGlu) return silu_glu(a0, a1);
  if (EPI == kSEpiRelu2) return relu2_f(a0);
  if (EPI == kSEpiTanh) return tanhf(a0);
  if (EPI == kSEpiDecaySoft) return decay_soft(a0 + bias, rate);
  if (EPI == kSEpiDecayExp) return decay_exp(a0 + bias);
  return a0 * p.scale;
}

template <int NTOK, int EPI>
__global__ void __launch_bounds__(kThreads, 1)
stack_gemm_kernel(const __grid_constant__ CUtensorMap tmW, const __grid_constant__ CUtensorMap tmW2,
                  const __grid_constant__ CUtensorMap tmX, const StackGemmArgs p, const int n_tiles, const int items,
                  const int row_tiles, const int items_fastest) {
  constexpr bool DUAL = EPI == kSEpiClampedGlu || EPI == kSEpiSiluGlu;
  using C = Cfg<NTOK, DUAL>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  Tail* tail = reinterpret_cast<Tail*>(smem + C::kStages * C::kStage);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kb_total = (p.k + kKStep - 1) / kKStep;

  if (threadIdx.x == 0) {
    for (int i = 0; i < C::kStages; ++i) { mbar_init(&tail->full[i], 1); mbar_init(&tail->empty[i], 1); }
    for (int i = 0; i < 2; ++i) { mbar_init(&tail->acc_full[i], 1); mbar_init(&tail->acc_empty[i], 256); }
    mbar_fence_init();
    tma_prefetch_desc(&tmW);
    tma_prefetch_desc(&tmX);
    if (DUAL) tma_prefetch_desc(&tmW2);
  }
  if (warp == 1) { tmem_alloc(&tail->tmem, C::kTmem); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tail->tmem;
  griddep_wait();
  griddep_launch();

  const int na = p.n_items ? min(min(*p.n_items, p.max_items), items) : items;
  const int total = n_tiles * items;
#define NRT_TILE(w, tile, item)                                    \
  const int tile = items_fastest ? (w) / items : (w) % n_tiles;    \
  const int item = items_fastest ? (w) % items : (w) / n_tiles;

  if (warp == 0) {
    if (elect_one()) {
      bool ok = true;
      int u = 0;
      for (int w = blockIdx.x; w < total && ok; w += gridDim.x) {
        NRT_TILE(w, tile, item)
        const Item it = item_of(p, item, row_tiles, NTOK, na);
        if (!it.live) continue;
        for (int kb = 0; kb < kb_total; ++kb, ++u) {
          const int st = u % C::kStages;
          if (u >= C::kStages && !mbar_wait(&tail->empty[st], ((u / C::kStages) & 1) ^ 1, p.status, kSiteStageEmpty | st)) { ok = false; break; }
          uint8_t* s = smem + st * C::kStage;
          mbar_expect_tx(&tail->full[st], C::kStage);
          tma_load_3d(s, &tmW, &tail->full[st], kb * kKStep, tile * kFeat, it.z);
          if (DUAL) tma_load_3d(s + kATile, &tmW2, &tail->full[st], kb * kKStep, tile * kFeat, it.z);
          tma_load_3d(s + (DUAL ? 2 : 1) * kATile, &tmX, &tail->full[st], kb * kKStep, p.n_items ? 0 : it.z, it.row0);
        }
      }
    }
  } else if (warp == 1) {
    if (elect_one()) {
      constexpr uint32_t idesc = umma_idesc(1u, kFeat, NTOK);
      bool ok = true;
      int u = 0, t = 0;
      for (int w = blockIdx.x; w < total && ok; w += gridDim.x) {
        NRT_TILE(w, tile, item)
        (void)tile;
        if (!item_of(p, item, row_tiles, NTOK, na).live) continue;
        const int buf = t & 1;
        if (t >= 2 && !mbar_wait(&tail->acc_empty[buf], ((t >> 1) & 1) ^ 1, p.status, kSiteAccEmpty | buf)) { ok = false; break; }
        tc_fence_after();
        for (int kb = 0; kb < kb_total; ++kb, ++u) {
          const int st = u % C::kStages;
          if (!mbar_wait(&tail->full[st], (u / C::kStages) & 1, p.status, kSiteTmaFull | st)) { ok = false; break; }
          tc_fence_after();
          const uint32_t s = smem_u32(smem + st * C::kStage);
          const uint64_t da = umma_desc_sw128(s), da2 = umma_desc_sw128(s + kATile);
          const uint64_t db = umma_desc_sw128(s + (DUAL ? 2 : 1) * kATile);
          const uint32_t d = tmem + buf * C::kAccCols;
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            umma_bf16(d, da + 2 * j, db + 2 * j, idesc, kb > 0 || j > 0);
            if (DUAL) umma_bf16(d + NTOK, da2 + 2 * j, db + 2 * j, idesc, kb > 0 || j > 0);
          }
          umma_commit(&tail->empty[st]);
          if (kb == kb_total - 1) umma_commit(&tail->acc_full[buf]);
        }
        ++t;
      }
    }
  } else {
    const int quad = warp & 3, half = (warp - 2) >> 2;
    const int feat = quad * 32 + lane;
    constexpr int kHalf = NTOK / 2;
    bool ok = true;
    int t = 0;
    for (int w = blockIdx.x; w < total && ok; w += gridDim.x) {
      NRT_TILE(w, tile, item)
      const Item it = item_of(p, item, row_tiles, NTOK, na);
      if (!it.live) continue;
      const int buf = t & 1;
      ok = __all_sync(0xffffffffu, mbar_wait(&tail->acc_full[buf], (t >> 1) & 1, p.status, kSiteAccFull | buf));
      if (!ok) break;
      tc_fence_after();
      const int n = tile * kFeat + feat;
      const bool live = n < p.n;
      const float bias = (epi_has_bias<EPI>() && live) ? bf(p.bias + (size_t)it.z * p.n + n) : 0.f;
      const float rate = (EPI == kSEpiDecaySoft && live) ? p.rate[n] : 0.f;
      const long long zoff = p.n_items ? 0 : it.z * p.out_zstride;
      const uint32_t acc = tmem + (uint32_t(quad * 32) << 16) + buf * C::kAccCols + half * kHalf;
      const int row_end = p.n_items ? 0x7fffffff : p.rows;
#pragma unroll 1
      for (int c = 0; c < kHalf; c += 32) {
        uint32_t v0[32], v1[DUAL ? 32 : 1];
        __syncwarp();                               // the loads below are warp-collective
        tmem_ld16_nowait(acc + c, v0);
        tmem_ld16_nowait(acc + c + 16, v0 + 16);
        if (DUAL) {
          tmem_ld16_nowait(acc + NTOK + c, v1);
          tmem_ld16_nowait(acc + NTOK + c + 16, v1 + (DUAL ? 16 : 0));
        }
        tmem_ld_wait();
        if (c + 32 == kHalf) {                      // last read of this accumulator: hand it back
          tc_fence_before();
          mbar_arrive(&tail->acc_empty[buf]);
        }
        const int row = it.row0 + half * kHalf + c;
        if (!live) {
        } else if (EPI == kSEpiTranspose) {
          // feature-major: the thread's 32 token columns are contiguous
          uint4* dst = reinterpret_cast<uint4*>(reinterpret_cast<__nv_bfloat16*>(p.out) + zoff + (long long)n * p.out_ld + row);
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            if (row + q * 8 < row_end) {
              uint4 o;
              o.x = pack_bf16x2(__uint_as_float(v0[q * 8]), __uint_as_float(v0[q * 8 + 1]));
              o.y = pack_bf16x2(__uint_as_float(v0[q * 8 + 2]), __uint_as_float(v0[q * 8 + 3]));
              o.z = pack_bf16x2(__uint_as_float(v0[q * 8 + 4]), __uint_as_float(v0[q * 8 + 5]));
              o.w = pack_bf16x2(__uint_as_float(v0[q * 8 + 6]), __uint_as_float(v0[q * 8 + 7]));
              dst[q] = o;
            }
          }
        } else {
          const long long at = (long long)row * p.out_ld + zoff + n;
          if (p.out_f32) {
            float* o = reinterpret_cast<float*>(p.out) + at;
#pragma unroll
            for (int r = 0; r < 32; ++r)
              if (row + r < row_end)
                o[(long long)r * p.out_ld] = epi_value<EPI>(p, __uint_as_float(v0[r]), DUAL ? __uint_as_float(v1[DUAL ? r : 0]) : 0.f, n, bias, rate);
          } else {
            __nv_bfloat16* o = reinterpret_cast<__nv_bfloat16*>(p.out) + at;
#pragma unroll
            for (int r = 0; r < 32; ++r)
              if (row + r < row_end)
                o[(long long)r * p.out_ld] = __float2bfloat16_rn(
                    epi_value<EPI>(p, __uint_as_float(v0[r]), DUAL ? __uint_as_float(v1[DUAL ? r : 0]) : 0.f, n, bias, rate));
          }
        }
      }
      ++t;
    }
  }
#undef NRT_TILE
  drain_on_error(p.status);
  tc_fence_before();
  __syncthreads();
  if (warp == 1) { tc_fence_after(); tmem_dealloc(tmem, C::kTmem); }
}

int sm_count() {
  static int sms = 0;
  if (!sms) {
    int dev = 0;
    cudaGetDevice(&dev);
    if (cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || sms < 1) sms = 148;
  }
  return sms;
}

template <int NTOK, int EPI>
int launch(const CUtensorMap& w, const CUtensorMap& w2, const CUtensorMap& x, const StackGemmArgs& a, int items_fastest,
           cudaStream_t stream) {
  constexpr bool DUAL = EPI == kSEpiClampedGlu || EPI == kSEpiSiluGlu;
  using C = Cfg<NTOK, DUAL>;
  auto* kern = stack_gemm_kernel<NTOK, EPI>;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, C::kSmem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const int n_tiles = (a.n + kFeat - 1) / kFeat;
  const int row_tiles = (a.rows + NTOK - 1) / NTOK;
  const int items = a.n_items ? a.max_items : a.zcount * row_tiles;
  if (items < 1 || n_tiles < 1 || (long long)items * n_tiles > 0x7fffffffLL) return -3;
  const int total = items * n_tiles, sms = sm_count();
  return launch_pdl(kern, dim3(total < sms ? total : sms), dim3(kThreads), C::kSmem, stream, false, w, w2, x, a, n_tiles, items,
                    row_tiles, items_fastest);
}

// ------------------------------------------------------------------------------------ float form
constexpr int kFT = 64, kFK = 16;             // 64 features x 64 rows per CTA, 4 x 4 per thread

template <int EPI>
__global__ void __launch_bounds__(256) stack_gemm_f32_kernel(const StackGemmArgs p, const int row_tiles) {
  constexpr bool DUAL = EPI == kSEpiClampedGlu || EPI == kSEpiSiluGlu;
  __shared__ float sw[kFK][kFT + 4], sw2[DUAL ? kFK : 1][kFT + 4], sx[kFK][kFT + 4];
  griddep_wait();
  griddep_launch();
  Item it;
  int row_lim;
  if (p.n_items) {
    // a segment may be taller than a tile: segments are cut into 64-row pieces
    const int per = (p.item_rows + kFT - 1) / kFT;
    const int item = blockIdx.y / per, part = blockIdx.y % per;
    it.live = item < min(*p.n_items, p.max_items);
    if (!it.live) return;
    it.z = p.item_z[item];
    row_lim = p.item_row[item] + p.item_rows;
    it.row0 = p.item_row[item] + part * kFT;
  } else {
    it = item_of(p, blockIdx.y, row_tiles, kFT, 0);
    row_lim = p.rows;
  }
  const int n0 = blockIdx.x * kFT;
  const float* X = reinterpret_cast<const float*>(p.act) + (p.n_items ? 0 : it.z * p.act_zstride);
  const __nv_bfloat16* W = p.w + it.z * p.w_zstride;
  const __nv_bfloat16* W2 = DUAL ? p.w2 + it.z * p.w_zstride : nullptr;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {}, acc2[4][4] = {};
  for (int k0 = 0; k0 < p.k; k0 += kFK) {
    for (int i = threadIdx.x; i < kFT * kFK; i += 256) {
      const int r = i / kFK, k = i % kFK;
      const bool kin = k0 + k < p.k;
      sw[k][r] = kin && n0 + r < p.n ? bf(W + (long long)(n0 + r) * p.w_ld + k0 + k) : 0.f;
      if (DUAL) sw2[k][r] = kin && n0 + r < p.n ? bf(W2 + (long long)(n0 + r) * p.w_ld + k0 + k) : 0.f;
      sx[k][r] = kin && it.row0 + r < row_lim ? X[(long long)(it.row0 + r) * p.act_ld + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kFK; ++k) {
      float xv[4], wv[4], w2v[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        xv[i] = sx[k][ty * 4 + i];
        wv[i] = sw[k][tx + 16 * i];
        w2v[i] = DUAL ? sw2[DUAL ? k : 0][tx + 16 * i] : 0.f;
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          acc[i][j] = fmaf(xv[i], wv[j], acc[i][j]);
          if (DUAL) acc2[i][j] = fmaf(xv[i], w2v[j], acc2[i][j]);
        }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int row = it.row0 + ty * 4 + i;
    if (row >= row_lim) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx + 16 * j;
      if (n >= p.n) continue;
      const float bias = epi_has_bias<EPI>() ? bf(p.bias + (size_t)it.z * p.n + n) : 0.f;
      const float rate = EPI == kSEpiDecaySoft ? p.rate[n] : 0.f;
      const float v = epi_value<EPI>(p, acc[i][j], acc2[i][j], n, bias, rate);
      store_act(p.out, (long long)row * p.out_ld + (p.n_items ? 0 : it.z * p.out_zstride) + n, v, p.out_f32);
    }
  }
}

template <int EPI>
int launch_f32(const StackGemmArgs& a, cudaStream_t stream) {
  const int row_tiles = (a.rows + kFT - 1) / kFT;
  const int items = a.n_items ? a.max_items * ((a.item_rows + kFT - 1) / kFT) : a.zcount * row_tiles;
  if (items < 1 || items > 65535) return -3;
  return launch_pdl(stack_gemm_f32_kernel<EPI>, dim3((a.n + kFT - 1) / kFT, items), dim3(256), 0, stream, false, a, row_tiles);
}

}  // namespace

extern "C" int nrt_stack_gemm_args_size() { return (int)sizeof(StackGemmArgs); }

// ntok: token rows per tile (64, 128, 256; two-product epilogues 64 or 128); the token map's box has that many rows.
extern "C" int nrt_stack_gemm(int epi, int ntok, const void* tmW, const void* tmW2, const void* tmX, const void* args,
                              int items_fastest, void* stream) {
  CUtensorMap w, w2, x;
  memcpy(&w, tmW, sizeof(w));
  memcpy(&w2, tmW2 ? tmW2 : tmW, sizeof(w2));
  memcpy(&x, tmX, sizeof(x));
  StackGemmArgs a;
  memcpy(&a, args, sizeof(a));
  if (a.n < 1 || a.k < 1 || a.rows < 1 || (a.n_items && a.item_rows != ntok)) return -3;
  if (((epi == kSEpiBias || epi == kSEpiDecaySoft || epi == kSEpiDecayExp) && !a.bias) || (epi == kSEpiDecaySoft && (!a.rate || a.zcount != 1))) return -3;
  if (epi == kSEpiTranspose && (a.out_f32 || a.out_ld % 8 || a.out_zstride % 8)) return -3;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
#define NRT_CASE(N, E) \
  if (ntok == N && epi == E) return launch<N, E>(w, w2, x, a, items_fastest, s);
  NRT_CASE(64, kSEpiStore) NRT_CASE(128, kSEpiStore) NRT_CASE(256, kSEpiStore)
  NRT_CASE(64, kSEpiBias) NRT_CASE(256, kSEpiBias)
  NRT_CASE(64, kSEpiTranspose) NRT_CASE(256, kSEpiTranspose)
  NRT_CASE(64, kSEpiClampedGlu) NRT_CASE(128, kSEpiClampedGlu)
  NRT_CASE(64, kSEpiSiluGlu) NRT_CASE(128, kSEpiSiluGlu)
  NRT_CASE(64, kSEpiRelu2) NRT_CASE(128, kSEpiRelu2) NRT_CASE(256, kSEpiRelu2)
  NRT_CASE(64, kSEpiTanh) NRT_CASE(256, kSEpiTanh)
  NRT_CASE(64, kSEpiDecaySoft) NRT_CASE(256, kSEpiDecaySoft)
  NRT_CASE(64, kSEpiDecayExp) NRT_CASE(256, kSEpiDecayExp)
#undef NRT_CASE
  return -2;
}

extern "C" int nrt_stack_gemm_f32(int epi, const void* args, void* stream) {
  StackGemmArgs a;
  memcpy(&a, args, sizeof(a));
  if (a.n < 1 || a.k < 1 || a.rows < 1) return -3;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  switch (epi) {
    case kSEpiStore: return launch_f32<kSEpiStore>(a, s);
    case kSEpiBias: return launch_f32<kSEpiBias>(a, s);
    case kSEpiClampedGlu: return launch_f32<kSEpiClampedGlu>(a, s);
    case kSEpiSiluGlu: return launch_f32<kSEpiSiluGlu>(a, s);
    case kSEpiRelu2: return launch_f32<kSEpiRelu2>(a, s);
    case kSEpiTanh: return launch_f32<kSEpiTanh>(a, s);
    case kSEpiDecaySoft: return launch_f32<kSEpiDecaySoft>(a, s);
    case kSEpiDecayExp: return launch_f32<kSEpiDecayExp>(a, s);
  }
  return -2;
}
