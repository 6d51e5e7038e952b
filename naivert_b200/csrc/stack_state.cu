// Mixers whose heads carry a matrix state: gated delta rule, bonus recurrence, normalised matrix memory.
//   chunk path   short convolution + SiLU + unit vectors (or mixes with the previous token), the recurrence over the chunk's rows,
//                read-out norm and gate
//   one token    one kernel: unit vectors, low-rank decay and gate, state update, read-out, norm and gate
//
// A value column of S evolves on its own given q, k and the decay, so columns are spread over the GPU; everything is fp32 (packed
// pairs).  Chunks go in blocks of eight tokens (stack.cuh): L lanes share four columns, lane l holds the 16-byte pieces l, l + L, ...
// of their dim entries in registers for the whole chunk; a block is two (delta: three) sets of independent products with the state and
// one update, with a single reduction over the lanes.  One token after the other, each with a reduction of its own, left a scheduler
// with one warp waiting for its own results two thirds of the time.
#include "stack.cuh"
#include "launch.hpp"

#include <string.h>

using namespace nrt;

namespace {

typedef unsigned long long u64;
constexpr int kLanes = 8;                     // lanes per value column
constexpr float kUnitEps = 1e-6f;             // added to the squared length of what becomes a unit vector

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

// ------------------------------------------------------------------------------------ chunk path: block records
// Running maximum of the normalised form over the whole chunk, one CTA per head: m -> max(f + m, i) composes as (sum of f, max).
constexpr int kScanT = 1024;

__global__ void __launch_bounds__(kScanT) gate_scan_kernel(const StateChunkArgs a) {
  __shared__ float wf[32], wb[32];
  griddep_wait();
  griddep_launch();
  const int h = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos0 = *a.pos0;
  const int slot = state_slot(a.tags, pos0, a.status);
  if (slot < 0) return;
  const long long m_at = (long long)a.heads * (a.vdim + 1) * pad4(a.dim) + h;
  float m = pos0 > 0 ? a.state[slot * a.state_stride + m_at] : 0.f;
  for (int r0 = 0; r0 < a.rows; r0 += kScanT) {
    const int r = r0 + threadIdx.x;
    const bool in = r < a.rows;
    const float zi = in ? log_input(a.gi[r * a.gate_ld + h], a.cap) : -FLT_MAX, zf = in ? log_forget(a.gf[r * a.gate_ld + h], a.cap) : 0.f;
    float f = zf, b = zi;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float fp = __shfl_up_sync(0xffffffffu, f, o), bp = __shfl_up_sync(0xffffffffu, b, o);
      if (lane >= o) {
        b = fmaxf(f + bp, b);
        f += fp;
      }
    }
    if (lane == 31) { wf[warp] = f; wb[warp] = b; }
    __syncthreads();
    float before = m;                          // running maximum ahead of this warp, then ahead of this token
    for (int w = 0; w < warp; ++w) before = fmaxf(wf[w] + before, wb[w]);
    const float mt = fmaxf(f + before, b);
    float mp = __shfl_up_sync(0xffffffffu, mt, 1);
    if (lane == 0) mp = before;
    if (in) {
      *reinterpret_cast<float2*>(a.keep + ((long long)r * a.heads + h) * 2) = make_float2(expf(zf + mp - mt), expf(zi - mt));
      a.den[((long long)r * a.heads + h) * 2 + 1] = expf(-mt);
    }
    for (int w = 0; w < kScanT / 32; ++w) m = fmaxf(wf[w] + m, wb[w]);
    __syncthreads();
  }
  if (threadIdx.x == 0) a.state[(1 - slot) * a.state_stride + m_at] = m;
}

// N values over the lanes -> N / L per lane: lane l keeps values N / L * l, ...
template <int N, int L>
__device__ __forceinline__ void scatter_sum(float (&v)[N], int l) {
#pragma unroll
  for (int o = L / 2, half = N / 2; o >= 1; o /= 2, half /= 2) {
    const bool up = l & o;
#pragma unroll
    for (int i = 0; i < N / 2; ++i)
      if (i < half) {
        const float keep = up ? v[i + half] : v[i], send = up ? v[i] : v[i + half];
        v[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
      }
  }
}

// One warp per (block, head); lane = key channels lane, lane + 32, ... of a slice.
template <int KIND, int NC>
__global__ void __launch_bounds__(128, 3) state_blocks_kernel(const StateChunkArgs a) {
  griddep_wait();
  griddep_launch();
  constexpr int B = kStateBlock;
  const int lane = threadIdx.x & 31, h = blockIdx.y * 4 + (threadIdx.x >> 5), r0 = blockIdx.x * B, n = min(B, a.rows - r0);
  if (h >= a.heads) return;
  const int hk = h / (a.heads / a.kv_heads), dp = state_row(a.dim);
  float* rec = a.blocks + ((long long)blockIdx.x * a.heads + h) * state_record(KIND, a.dim);
  float* k1 = rec;                             // (delta)
  float* q1 = rec + (KIND == kStateDelta ? B * dp : 0);
  float* k2 = q1 + B * dp;
  float* whole = k2 + B * dp;
  float* pairs = whole + dp;
  float keep[B], add[B];
#pragma unroll
  for (int t = 0; t < B; ++t) {
    keep[t] = add[t] = 1.f;
    if (KIND == kStateNormalized && t < n) {
      const float2 c = *reinterpret_cast<const float2*>(a.keep + ((long long)(r0 + t) * a.heads + h) * 2);
      keep[t] = c.x;
      add[t] = c.y;
    }
  }
  float w[B * B];                              // pair coefficients, partial sums
#pragma unroll
  for (int i = 0; i < B * B; ++i) w[i] = 0.f;
  for (int d0 = 0; d0 < dp; d0 += 32 * NC) {
    float q[B][NC], k[B][NC], g[B][NC];
    // loads without conditions (clamped addresses), so that all of them are in flight together
#pragma unroll
    for (int t = 0; t < B; ++t)
#pragma unroll
      for (int i = 0; i < NC; ++i) {
        const int d = min(d0 + lane + 32 * i, a.dim - 1);
        const long long r = min(r0 + t, a.rows - 1);
        q[t][i] = __ldg(a.q + r * a.q_ld + hk * a.dim + d);
        k[t][i] = __ldg(a.k + r * a.k_ld + hk * a.dim + d);
        g[t][i] = KIND == kStateNormalized ? keep[t] : __ldg(a.g + r * a.g_ld + h * a.dim + d);
      }
#pragma unroll
    for (int t = 0; t < B; ++t)
#pragma unroll
      for (int i = 0; i < NC; ++i) {
        const bool in = t < n && d0 + lane + 32 * i < a.dim;
        q[t][i] = in ? q[t][i] * a.q_scale : 0.f;
        k[t][i] = in ? k[t][i] : 0.f;
        if (KIND != kStateNormalized && !in) g[t][i] = 1.f;
      }
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int d = d0 + lane + 32 * i;
      float c = 1.f;
#pragma unroll
      for (int t = 0; t < B; ++t) {
        if (KIND == kStateBonus) q1[t * dp + d] = c * q[t][i];            // the read-out sees the state ahead of the token
        c *= g[t][i];
        if (KIND != kStateBonus) q1[t * dp + d] = c * q[t][i];
        if (KIND == kStateDelta) k1[t * dp + d] = c * k[t][i];
      }
      whole[d] = c;
      c = 1.f;
#pragma unroll
      for (int t = B - 1; t >= 0; --t) {
        k2[t * dp + d] = c * add[t] * k[t][i];
        c *= g[t][i];
      }
      const float bonus = KIND == kStateBonus && d < a.dim ? bf(a.u + (long long)h * a.dim + d) : 1.f;
#pragma unroll
      for (int s = 0; s < B; ++s) {
        c = k[s][i] * add[s];
        w[s * B + s] = fmaf(q[s][i], c * bonus, w[s * B + s]);
#pragma unroll
        for (int t = s + 1; t < B; ++t) {
          if (KIND == kStateBonus) w[t * B + s] = fmaf(q[t][i], c, w[t * B + s]);
          c *= g[t][i];
          if (KIND != kStateBonus) w[t * B + s] = fmaf(q[t][i], c, w[t * B + s]);
          if (KIND == kStateDelta) w[s * B + t] = fmaf(k[t][i], c, w[s * B + t]);
        }
      }
    }
  }
  scatter_sum<B * B, 32>(w, lane);
  *reinterpret_cast<float2*>(pairs + 2 * lane) = make_float2(w[0], w[1]);
  if (lane < B) pairs[B * B + lane] = KIND == kStateDelta && lane < n ? sigmoid_f(a.beta[(r0 + lane) * a.beta_ld + h]) : 0.f;
}

// ------------------------------------------------------------------------------------ chunk path: the recurrence
// grid (column tiles, heads, pieces); a warp holds 4 * 32 / L columns; records and values arrive three stages deep, the records as one
// bulk copy.  Recurrences that are linear in the state are cut into pieces of the chunk: a first launch (SUMS) leaves each piece's end
// state from zero and its decay, the second starts every piece from the carried state and the earlier pieces' sums.
constexpr int kQuad = 4, kStages = 3;

template <int L, int NV>
__device__ __forceinline__ void state_products(const u64 (&s)[kQuad][2 * NV], const ulonglong2* vec, float (&out)[32]) {
  // out[value]: value = 32 / L * lane + i belongs to column lane & 3 and token (lane >> 2) + L / 4 * i
  constexpr int VPL = 32 / L;
  u64 acc[kStateBlock][kQuad];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    ulonglong2 x[kStateBlock];
#pragma unroll
    for (int t = 0; t < kStateBlock; ++t) x[t] = vec[t * (NV * L) + i * L];
#pragma unroll
    for (int t = 0; t < kStateBlock; ++t)
#pragma unroll
      for (int j = 0; j < kQuad; ++j) acc[t][j] = i == 0 ? mul2(s[j][0], x[t].x) : fma2(s[j][2 * i], x[t].x, acc[t][j]);
#pragma unroll
    for (int t = 0; t < kStateBlock; ++t)
#pragma unroll
      for (int j = 0; j < kQuad; ++j) acc[t][j] = fma2(s[j][2 * i + 1], x[t].y, acc[t][j]);
  }
#pragma unroll
  for (int v = 0; v < 32; ++v) out[v] = both(acc[(v / VPL >> 2) + L / 4 * (v % VPL)][v / VPL & 3]);
}

template <int KIND, int L, int NV, bool SUMS>
__global__ void __launch_bounds__(256, 1) state_chunk_kernel(const StateChunkArgs a, const int piece_blocks) {
  constexpr int B = kStateBlock, DP = NV * 4 * L, PER_WARP = 32 / L * kQuad, VPL = 32 / L;
  constexpr int ROWS = (KIND == kStateDelta ? 3 : 2) * B, RECORD = (ROWS + 1) * DP + B * B + B;
  constexpr int SKIP = SUMS ? (ROWS - B) * DP : 0, REC = SUMS ? (B + 1) * DP : RECORD;      // the part of a record that is read
  constexpr int K2 = SUMS ? 0 : (ROWS - B) * DP, WHOLE = K2 + B * DP;
  extern __shared__ __align__(16) float sh[];
  __shared__ uint64_t full[kStages];
  griddep_wait();
  griddep_launch();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, l = lane & (L - 1);
  const int cols = (blockDim.x >> 5) * PER_WARP, C = a.vdim + extra_columns<KIND>(), d4 = pad4(a.dim);
  const int h = blockIdx.y, c0 = blockIdx.x * cols, c = c0 + warp * PER_WARP + lane / L * kQuad;
  const int pos0 = *a.pos0;
  const int slot = state_slot(a.tags, pos0, a.status);
  if (slot < 0) return;
  const float* old = a.state + slot * a.state_stride;
  float* now = a.state + (1 - slot) * a.state_stride;
  const long long at = ((long long)h * C + c) * d4;

  u64 s[kQuad][2 * NV];
#pragma unroll
  for (int j = 0; j < kQuad; ++j)
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      ulonglong2 v = make_ulonglong2(0ull, 0ull);
      const int e = (l + L * i) * 4;
      if (!SUMS && c + j < C && pos0 > 0 && e < d4) v = *reinterpret_cast<const ulonglong2*>(old + at + (long long)j * d4 + e);
      s[j][2 * i] = v.x;
      s[j][2 * i + 1] = v.y;
    }
  const int piece = blockIdx.z;
  float* decays = a.sums + (long long)(kStatePieces - 1) * a.heads * C * d4;
  u64 kept[2 * NV];                            // SUMS: the piece's decay so far
#pragma unroll
  for (int i = 0; i < 2 * NV; ++i) kept[i] = pack2(1.f, 1.f);
  if (!SUMS && KIND != kStateDelta)
    for (int z = 0; z < piece; ++z) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int e = (l + L * i) * 4;
        if (e >= d4) continue;
        const ulonglong2 g = *reinterpret_cast<const ulonglong2*>(decays + ((long long)z * a.heads + h) * d4 + e);
#pragma unroll
        for (int j = 0; j < kQuad; ++j)
          if (c + j < C) {
            const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(a.sums + (((long long)z * a.heads + h) * C + c + j) * d4 + e);
            s[j][2 * i] = fma2(s[j][2 * i], g.x, v.x);
            s[j][2 * i + 1] = fma2(s[j][2 * i + 1], g.y, v.y);
          }
      }
    }

  float* sv = sh + kStages * REC;                                        // [stages][B][cols]
  float* work = sv + kStages * B * cols + (warp * (32 / L) + lane / L) * 2 * B * kQuad;     // this lane group's: S^T k, updates [B][4]
  for (int i = threadIdx.x; i < kStages * B * cols; i += blockDim.x) {
    const int cc = c0 + i % cols;
    sv[i] = KIND == kStateNormalized && cc == a.vdim ? 1.f : 0.f;         // the normaliser's column
  }
  if (threadIdx.x == 0) {
    for (int i = 0; i < kStages; ++i) mbar_init(&full[i], 1);
    mbar_fence_init();
  }
  __syncthreads();
  const int b0 = piece * piece_blocks, blocks = min((a.rows + B - 1) / B, b0 + piece_blocks);
  const float* v0 = a.v + (long long)h * a.vdim + c0;
  const int vcols = min(cols, a.vdim - c0);                              // (none in a tile that holds only the normaliser)
  const bool quads = vcols > 0 && ((reinterpret_cast<uintptr_t>(v0) & 15) | (uintptr_t)((a.v_ld | vcols) & 3)) == 0;
  const int step = quads ? 4 : 1, per = max(vcols, 0) / step;
  auto request = [&](int b, int st) {
    if (threadIdx.x == 0) {
      mbar_expect_tx(&full[st], REC * 4);
      asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                   ::"r"(smem_u32(sh + st * REC)), "l"(a.blocks + ((long long)b * a.heads + h) * RECORD + SKIP), "r"(REC * 4), "r"(smem_u32(&full[st]))
                   : "memory");
    }
    const int n = min(B, a.rows - b * B);
    for (int i = threadIdx.x; i < n * per; i += blockDim.x) {
      const int t = i / per, e = (i - t * per) * step;
      const uint32_t dst = smem_u32(sv + (st * B + t) * cols + e);
      const float* src = v0 + (b * B + t) * a.v_ld + e;
      if (quads) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
      else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(dst), "l"(src) : "memory");
    }
  };
  if (b0 < blocks) request(b0, 0);
  asm volatile("cp.async.commit_group;" ::: "memory");
  if (b0 + 1 < blocks) request(b0 + 1, 1);
  asm volatile("cp.async.commit_group;" ::: "memory");
  const int col = l & 3, tq = l >> 2;                                    // this lane's column and first token among the reduced values
  bool ok = true;
  for (int b = b0, st = 0; b < blocks; ++b, st = st + 1 == kStages ? 0 : st + 1) {
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    ok = __syncthreads_and(mbar_wait(&full[st], ((b - b0) / kStages) & 1, a.status, kSiteTmaFull | st));
    if (!ok) break;
    if (b + 2 < blocks) request(b + 2, st + 2 >= kStages ? st + 2 - kStages : st + 2);       // (its last reader has passed the barrier)
    asm volatile("cp.async.commit_group;" ::: "memory");
    const float* rec = sh + st * REC;
    const ulonglong2* vec = reinterpret_cast<const ulonglong2*>(rec) + l;
    const float* pairs = rec + (ROWS + 1) * DP;
    const float* vc = sv + st * B * cols + (c - c0);
    float p[32], q[32];
    if (KIND == kStateDelta) {
      state_products<L, NV>(s, vec, p);
      scatter_sum<32, L>(p, l);
#pragma unroll
      for (int i = 0; i < VPL; ++i) work[(tq + L / 4 * i) * kQuad + col] = p[i];
    }
    if (!SUMS) {
      state_products<L, NV>(s, vec + (KIND == kStateDelta ? B * DP / 4 : 0), q);
      scatter_sum<32, L>(q, l);
    }
    const float* upd = vc;                     // the tokens' updates of the group's columns, rows of `upd_ld`
    int upd_ld = cols;
    if (KIND == kStateDelta) {
      __syncwarp();
      float* us = work + B * kQuad;
      if (l < kQuad) {
        float r[B];
#pragma unroll
        for (int t = 0; t < B; ++t) r[t] = vc[t * cols + col] - work[t * kQuad + col];
#pragma unroll
        for (int t = 0; t < B; ++t) {
          const float u = pairs[B * B + t] * r[t];
          us[t * kQuad + col] = u;
          const float4 w0 = *reinterpret_cast<const float4*>(pairs + t * B), w1 = *reinterpret_cast<const float4*>(pairs + t * B + 4);
          const float w[B] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
          for (int x = t + 1; x < B; ++x) r[x] = fmaf(-w[x], u, r[x]);
        }
      }
      __syncwarp();
      upd = us;
      upd_ld = kQuad;
    }
    // the state moves on by the whole block
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const ulonglong2 g = vec[WHOLE / 4 + i * L];
      if (SUMS) {
        kept[2 * i] = mul2(kept[2 * i], g.x);
        kept[2 * i + 1] = mul2(kept[2 * i + 1], g.y);
      }
#pragma unroll
      for (int j = 0; j < kQuad; ++j) {
        s[j][2 * i] = mul2(s[j][2 * i], g.x);
        s[j][2 * i + 1] = mul2(s[j][2 * i + 1], g.y);
      }
    }
#pragma unroll
    for (int t = 0; t < B; ++t) {
      const float4 u = *reinterpret_cast<const float4*>(upd + t * upd_ld);
      const u64 uu[kQuad] = {pack2(u.x, u.x), pack2(u.y, u.y), pack2(u.z, u.z), pack2(u.w, u.w)};
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const ulonglong2 k = vec[(K2 + t * DP) / 4 + i * L];
#pragma unroll
        for (int j = 0; j < kQuad; ++j) {
          s[j][2 * i] = fma2(k.x, uu[j], s[j][2 * i]);
          s[j][2 * i + 1] = fma2(k.y, uu[j], s[j][2 * i + 1]);
        }
      }
    }
    if (SUMS) continue;
    // read-outs: this lane's column at its tokens
    float uc[B];
#pragma unroll
    for (int e = 0; e < B; ++e) uc[e] = upd[e * upd_ld + col];
#pragma unroll
    for (int i = 0; i < VPL; ++i) {
      const int t = tq + L / 4 * i;
      const float4 w0 = *reinterpret_cast<const float4*>(pairs + t * B), w1 = *reinterpret_cast<const float4*>(pairs + t * B + 4);
      const float w[B] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
      float x = q[i], x1 = 0.f;
#pragma unroll
      for (int e = 0; e < B; e += 2) {
        x = fmaf(e <= t ? w[e] : 0.f, uc[e], x);
        x1 = fmaf(e + 1 <= t ? w[e + 1] : 0.f, uc[e + 1], x1);
      }
      x += x1;
      const int r = b * B + t;
      if (r < a.rows) {
        if (c + col < a.vdim) a.o[((long long)r * a.heads + h) * a.vdim + c + col] = x;
        else if (KIND == kStateNormalized && c + col == a.vdim) a.den[((long long)r * a.heads + h) * 2] = x;
      }
    }
    if (KIND == kStateDelta) __syncwarp();                               // the work area is rewritten
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  if (!ok) {
    drain_on_error(a.status);
    return;
  }
  if (!SUMS && piece != (int)gridDim.z - 1) return;
  float* end = SUMS ? a.sums + ((long long)piece * a.heads + h) * C * d4 + (long long)c * d4 : now + at;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int e = (l + L * i) * 4;
    if (e >= d4) continue;
#pragma unroll
    for (int j = 0; j < kQuad; ++j)
      if (c + j < C) *reinterpret_cast<ulonglong2*>(end + (long long)j * d4 + e) = make_ulonglong2(s[j][2 * i], s[j][2 * i + 1]);
    if (SUMS && blockIdx.x == 0 && threadIdx.x < L)
      *reinterpret_cast<ulonglong2*>(decays + ((long long)piece * a.heads + h) * d4 + e) = make_ulonglong2(kept[2 * i], kept[2 * i + 1]);
  }
  if (SUMS) return;
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
constexpr int kConvStrip = 16, kConvWin = 4;  // rows per warp; taps that stay in a register window (longer kernels re-read their inputs)

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
  auto input = [&](int rr, int c) {            // row rr of the projection, or what earlier chunks left
    if (rr >= 0) return __ldg(a.proj + rr * a.ld + col + c);
    return pos0 + rr >= 0 ? a.history[(long long)((pos0 + rr) % a.hist_rows) * columns + col + c] : 0.f;
  };
  auto finish = [&](int r, float (&y)[NC]) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      y[i] = lane + 32 * i < w ? silu_f(y[i]) : 0.f;
      ss = fmaf(y[i], y[i], ss);
    }
    const float scale = is_v ? 1.f : (seg < G ? a.q_scale : 1.f) / sqrtf(lane_sum(ss) + kUnitEps);
#pragma unroll
    for (int i = 0; i < NC; ++i)
      if (lane + 32 * i < w) out[r * out_ld + lane + 32 * i] = y[i] * scale;
  };
  if (a.taps <= kConvWin) {
    constexpr int BATCH = NC <= 4 ? 4 : 1;     // rows requested together
    float kw[NC][kConvWin], x[NC][kConvWin];   // newest last; missing taps are zero
#pragma unroll
    for (int i = 0; i < NC; ++i)
#pragma unroll
      for (int j = 0; j < kConvWin; ++j) {
        const int c = lane + 32 * i, t = j - (kConvWin - a.taps);
        kw[i][j] = c < w && t >= 0 ? bf(kern + c * a.taps + t) : 0.f;
        x[i][j] = c < w && j > kConvWin - a.taps ? input(r0 - (kConvWin - j), c) : 0.f;
      }
#pragma unroll 1
    for (int rb = r0; rb < r1; rb += BATCH) {
      float in[BATCH][NC];
#pragma unroll
      for (int q = 0; q < BATCH; ++q)
#pragma unroll
        for (int i = 0; i < NC; ++i) in[q][i] = rb + q < r1 && lane + 32 * i < w ? __ldg(a.proj + (rb + q) * a.ld + col + lane + 32 * i) : 0.f;
#pragma unroll
      for (int q = 0; q < BATCH; ++q) {
        if (rb + q >= r1) break;
        float y[NC];
#pragma unroll
        for (int i = 0; i < NC; ++i) {
          y[i] = 0.f;
#pragma unroll
          for (int j = 0; j < kConvWin; ++j) {
            x[i][j] = j + 1 < kConvWin ? x[i][j + 1] : in[q][i];
            y[i] = fmaf(kw[i][j], x[i][j], y[i]);
          }
        }
        finish(rb + q, y);
      }
    }
    return;
  }
  for (int r = r0; r < r1; ++r) {
    float y[NC];
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = lane + 32 * i;
      y[i] = 0.f;
      if (c < w)
        for (int j = 0; j < a.taps; ++j) y[i] = fmaf(bf(kern + c * a.taps + j), input(r - (a.taps - 1 - j), c), y[i]);
    }
    finish(r, y);
  }
}

__device__ __forceinline__ float4 bf4(const __nv_bfloat16* p) {
  const uint2 v = __ldg(reinterpret_cast<const uint2*>(p));
  return make_float4(bf16_lo(v.x), bf16_hi(v.x), bf16_lo(v.y), bf16_hi(v.y));
}
__device__ __forceinline__ void store_act4(void* base, long long i, const float4& v, int f32) {
  if (f32) *reinterpret_cast<float4*>(reinterpret_cast<float*>(base) + i) = v;
  else *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(base) + i) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
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
  if (((a.width | (int)a.out_ld | (int)a.state_stride) & 3) == 0 && (reinterpret_cast<uintptr_t>(a.shift) & 15) == 0) {
    for (int c = threadIdx.x * 4; c < a.width; c += 1024) {
      const float4 v = __ldg(reinterpret_cast<const float4*>(x + c));
      const float4 b = before ? *reinterpret_cast<const float4*>(before + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      const float4 d = make_float4(b.x - v.x, b.y - v.y, b.z - v.z, b.w - v.w);
#pragma unroll 5
      for (int s = 0; s < a.mixes; ++s) {
        const float4 m = bf4(a.mu + (long long)s * a.width + c);
        store_act4(a.out, o0 + s * a.out_ld + c, make_float4(fmaf(d.x, m.x, v.x), fmaf(d.y, m.y, v.y), fmaf(d.z, m.z, v.z), fmaf(d.w, m.w, v.w)), a.f32);
      }
      if (keep) *reinterpret_cast<float4*>(keep + c) = v;
    }
    return;
  }
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
  const float* g = a.gate + (long long)r * a.gate_ld + (long long)h * a.vdim;
  const __nv_bfloat16* w = a.norm + (a.norm_per_head ? (long long)h * a.vdim : 0);
  const long long at = (long long)r * a.out_ld + (long long)h * a.vdim;
  auto gated = [&](float z) { return a.gate_kind == kGateSilu ? silu_f(z) : sigmoid_f(z); };
  float ss = 0.f;
  if (((a.vdim | (int)a.gate_ld | (int)a.out_ld) & 3) == 0 && (reinterpret_cast<uintptr_t>(a.gate) & 15) == 0) {
    constexpr int KEEP = 4;                    // pieces of a head that stay in registers between the two passes
    float4 keep[KEEP], z[KEEP];
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int c = (lane + 32 * i) * 4;
      keep[i] = z[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < a.vdim) {
        keep[i] = __ldg(reinterpret_cast<const float4*>(o + c));
        z[i] = __ldg(reinterpret_cast<const float4*>(g + c));
      }
    }
    auto sq = [&](const float4& v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; };
    auto put = [&](int c, const float4& v, const float4& zz, float rs) {
      const float4 n = bf4(w + c);
      store_act4(a.out, at + c, make_float4(v.x * rs * n.x * gated(zz.x), v.y * rs * n.y * gated(zz.y), v.z * rs * n.z * gated(zz.z), v.w * rs * n.w * gated(zz.w)), a.f32);
    };
#pragma unroll
    for (int i = 0; i < KEEP; ++i) ss += sq(keep[i]);
    for (int c = (lane + 32 * KEEP) * 4; c < a.vdim; c += 128) ss += sq(__ldg(reinterpret_cast<const float4*>(o + c)));
    const float rs = inv / sqrtf(lane_sum(ss) * inv * inv / (float)a.vdim + a.eps);
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
      if ((lane + 32 * i) * 4 < a.vdim) put((lane + 32 * i) * 4, keep[i], z[i], rs);
    for (int c = (lane + 32 * KEEP) * 4; c < a.vdim; c += 128) put(c, __ldg(reinterpret_cast<const float4*>(o + c)), __ldg(reinterpret_cast<const float4*>(g + c)), rs);
    return;
  }
  for (int c = lane; c < a.vdim; c += 32) {
    const float v = __ldg(o + c) * inv;
    ss = fmaf(v, v, ss);
  }
  const float rs = inv / sqrtf(lane_sum(ss) / (float)a.vdim + a.eps);
  for (int c = lane; c < a.vdim; c += 32) store_act(a.out, at + c, __ldg(o + c) * rs * bf(w + c) * gated(__ldg(g + c)), a.f32);
}

// ------------------------------------------------------------------------------------ one token
// grid (share of the value columns, heads); the CTAs of a head are a cluster that meets once, for the read-out norm.  The state (written
// a whole step ago) and the low-rank weights are requested before the wait for the predecessor.  Every instruction runs about once, so
// the kernel is bound by latencies, instruction fetch among them: loops stay rolled and nothing is specialised twice.
constexpr int kStepT = 256, kStepCols = kStepT / kLanes;

__device__ __forceinline__ void stage_weights(void* dst, const __nv_bfloat16* src, int n) {        // n a multiple of 8
#pragma unroll 1
  for (int i = threadIdx.x * 8; i < n; i += kStepT * 8)
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(reinterpret_cast<__nv_bfloat16*>(dst) + i)), "l"(src + i) : "memory");
}
// out[row] = W[row] . in for rows of ld bf16 (a multiple of 8), eight lanes per row
__device__ __forceinline__ void low_rank_rows(const __nv_bfloat16* w, int ld, int rows, const float* in, float* out) {
  const int l = threadIdx.x & (kLanes - 1);
#pragma unroll 1
  for (int rb = 0; rb < rows; rb += kStepT / kLanes) {                   // (the same trip count for every lane of a warp)
    const int r = rb + (threadIdx.x / kLanes);
    float acc = 0.f;
    if (r < rows) {
#pragma unroll 2
      for (int c = l * 8; c < ld; c += 8 * kLanes) {
        const uint4 p = *reinterpret_cast<const uint4*>(w + (long long)r * ld + c);
        const float4 x = *reinterpret_cast<const float4*>(in + c), y = *reinterpret_cast<const float4*>(in + c + 4);
        acc = fmaf(bf16_lo(p.x), x.x, fmaf(bf16_hi(p.x), x.y, fmaf(bf16_lo(p.y), x.z, fmaf(bf16_hi(p.y), x.w, acc))));
        acc = fmaf(bf16_lo(p.z), y.x, fmaf(bf16_hi(p.z), y.y, fmaf(bf16_lo(p.w), y.z, fmaf(bf16_hi(p.w), y.w, acc))));
      }
    }
    acc = column_sum(acc);
    if (r < rows && l == 0) out[r] = acc;
  }
}
__host__ __device__ inline int step_floats(int dp, int per, int decay_ld, int gate_ld) { return 3 * dp + 3 * pad4(per) + decay_ld + gate_ld; }

template <int KIND, int NV>
__global__ void __launch_bounds__(kStepT, 1) state_step_kernel(const StateStepArgs a, const int per, const int staged) {
  constexpr int DP = NV * 4 * kLanes;
  extern __shared__ __align__(16) float sh[];
  __shared__ float red[33], part;
  const int rank = blockIdx.x, h = blockIdx.y, hk = h / (a.heads / a.kv_heads);
  const int c_lo = min(a.vdim, rank * per), own = min(a.vdim, c_lo + per) - c_lo;
  const int decay_ld = (int)a.decay_ld, gate_ld = (int)a.gate_ld;
  float* sk = sh;
  float* sq = sk + DP;
  float* sg = sq + DP;
  float* so = sg + DP;
  float* sgate = so + pad4(per);
  float* sv = sgate + pad4(per);
  float* slow = sv + pad4(per);
  float* sgin = slow + decay_ld;
  const __nv_bfloat16* wdecay = KIND == kStateNormalized ? nullptr : a.decay_w + (long long)h * a.dim * decay_ld;
  const __nv_bfloat16* wgate = a.gate_w ? a.gate_w + ((long long)h * a.vdim + c_lo) * gate_ld : nullptr;
  const int tid = threadIdx.x, lane = tid & 31, l = lane & (kLanes - 1);
  const int C = a.vdim + extra_columns<KIND>(), d4 = pad4(a.dim);
  if (staged) {
    __nv_bfloat16* sw = reinterpret_cast<__nv_bfloat16*>(sgin + gate_ld);
    if (KIND != kStateNormalized) {
      stage_weights(sw, wdecay, a.dim * decay_ld);
      wdecay = sw;
      sw += a.dim * decay_ld;
    }
    if (a.gate_w) {
      stage_weights(sw, wgate, own * gate_ld);
      wgate = sw;
    }
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  const int pos = *reinterpret_cast<const volatile int*>(a.pos0);
  const int slot = state_slot(a.tags, pos, a.status);
  const float* old = a.state + max(slot, 0) * a.state_stride + (long long)h * C * d4;
  float* now = a.state + (1 - max(slot, 0)) * a.state_stride + (long long)h * C * d4;
  u64 s[2 * NV];
  auto load = [&](int j) {                     // local value column j
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int e = (l + kLanes * i) * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (j < own && pos > 0 && e < d4) v = __ldcg(reinterpret_cast<const float4*>(old + (long long)(c_lo + j) * d4 + e));
      s[2 * i] = pack2(v.x, v.y);
      s[2 * i + 1] = pack2(v.z, v.w);
    }
  };
  load(tid / kLanes);
  float d_bias = 0.f, d_rate = 0.f, norm = 0.f, n_old = 0.f;              // of this thread's first decay, column and normaliser entry
  if (KIND != kStateNormalized && tid < a.dim) {
    d_bias = bf(a.decay_b + (long long)h * a.dim + tid);
    if (a.rate) d_rate = __ldg(a.rate + (long long)h * a.dim + tid);
  }
  const __nv_bfloat16* nw = a.norm + (a.norm_per_head ? (long long)h * a.vdim : 0) + c_lo;
  if (tid < own) norm = bf(nw + tid);
  if (KIND == kStateNormalized && tid < a.dim && pos > 0) n_old = __ldcg(old + (long long)a.vdim * d4 + tid);
  griddep_wait();
  griddep_launch();
  if (slot >= 0) {                                                       // (the same for every CTA of the cluster)
    const float* p = a.proj;
    float s0 = 0.f, s1 = 0.f, floor_n = 0.f;
    if (KIND == kStateDelta) s0 = __ldcg(p + a.beta_off + h);
    if (KIND == kStateNormalized) { s0 = __ldcg(p + a.gi_off + h); s1 = __ldcg(p + a.gf_off + h); }
    float qq = 0.f, kk = 0.f, bonus = 0.f;
#pragma unroll 1
    for (int i = tid; i < DP; i += kStepT) {
      const bool in = i < a.dim;
      const float k = in ? __ldcg(p + a.k_off + hk * a.dim + i) : 0.f, q = in ? __ldcg(p + a.q_off + hk * a.dim + i) : 0.f;
      sk[i] = k;
      sq[i] = q;
      sg[i] = 0.f;
      if (KIND == kStateDelta) {
        qq = fmaf(q, q, qq);
        kk = fmaf(k, k, kk);
      }
      if (KIND == kStateBonus && in) bonus = fmaf(q * bf(a.u + (long long)h * a.dim + i), k, bonus);
    }
#pragma unroll 1
    for (int j = tid; j < own; j += kStepT) {
      sv[j] = __ldcg(p + a.v_off + (long long)h * a.vdim + c_lo + j);
      if (!a.gate_w) sgate[j] = __ldcg(p + a.gate_off + (long long)h * a.vdim + c_lo + j);
    }
    if (KIND != kStateNormalized) {
#pragma unroll 1
      for (int i = tid; i < decay_ld; i += kStepT) {
        const float z = i < a.low_rank ? __ldcg(p + a.low_off + i) : 0.f;
        slow[i] = a.low_tanh ? tanhf(z) : z;
      }
    }
    if (a.gate_w) {
#pragma unroll 1
      for (int i = tid; i < gate_ld; i += kStepT) sgin[i] = i < a.gate_rank ? __ldcg(p + a.gate_off + i) : 0.f;
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (KIND != kStateNormalized) low_rank_rows(wdecay, decay_ld, a.dim, slow, sg);
    if (a.gate_w) low_rank_rows(wgate, gate_ld, own, sgin, sgate);
    float q_scale = a.q_scale, k_scale = 1.f;
    if (KIND == kStateDelta) {
      s0 = sigmoid_f(s0);
      if (a.unit) {
        q_scale /= sqrtf(block_sum_f(qq, red) + kUnitEps);
        k_scale = 1.0f / sqrtf(block_sum_f(kk, red) + kUnitEps);
      }
    }
    if (KIND == kStateBonus) bonus = block_sum_f(bonus, red);
    if (KIND == kStateNormalized) {
      const float zi = log_input(s0, a.cap), zf = log_forget(s1, a.cap);
      const long long m_at = (long long)(a.heads - h) * C * d4 + h;      // the maxima follow the last head's state
      const float m = pos > 0 ? __ldcg(old + m_at) : 0.f, m_new = fmaxf(zf + m, zi);
      s0 = expf(zf + m - m_new);
      s1 = expf(zi - m_new);
      floor_n = expf(-m_new);
      if (rank == 0 && tid == 0) now[m_at] = m_new;
      // the normaliser: every CTA needs n . q, one keeps n
      float nq = 0.f;
#pragma unroll 1
      for (int d = tid; d < a.dim; d += kStepT) {
        const float n = fmaf(s0, d == tid ? n_old : pos > 0 ? __ldcg(old + (long long)a.vdim * d4 + d) : 0.f, s1 * sk[d]);
        nq = fmaf(n, sq[d], nq);
        if (rank == 0) now[(long long)a.vdim * d4 + d] = n;
      }
      q_scale /= fmaxf(fabsf(block_sum_f(nq, red) * q_scale), floor_n) + 1e-6f;
    } else {
      __syncthreads();                                                   // the low-rank results
#pragma unroll 1
      for (int d = tid; d < a.dim; d += kStepT) {
        const float z = sg[d] + (d == tid ? d_bias : bf(a.decay_b + (long long)h * a.dim + d));
        sg[d] = a.rate ? decay_soft(z, d == tid ? d_rate : a.rate[(long long)h * a.dim + d]) : decay_exp(z);
        if (KIND == kStateDelta) sk[d] *= k_scale;
      }
      __syncthreads();
    }
    const ulonglong2* q = reinterpret_cast<const ulonglong2*>(sq) + l;
    const ulonglong2* k = reinterpret_cast<const ulonglong2*>(sk) + l;
    const ulonglong2* g = reinterpret_cast<const ulonglong2*>(sg) + l;
    float ss = 0.f;
#pragma unroll 1
    for (int jb = 0; jb < own; jb += kStepCols) {                        // (the same trip count for every lane of a warp)
      const int j = jb + tid / kLanes;
      if (jb > 0) load(j);
      const float v = j < own ? sv[j] : 0.f;
      float r = column_sum(column_step<KIND, NV>(s, q, k, g, v, s0, s1));
      if (KIND == kStateBonus) r = fmaf(bonus, v, r);
      r *= q_scale;
      if (j < own) {
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          const int e = (l + kLanes * i) * 4;
          if (e < d4) *reinterpret_cast<ulonglong2*>(now + (long long)(c_lo + j) * d4 + e) = make_ulonglong2(s[2 * i], s[2 * i + 1]);
        }
        if (l == 0) {
          so[j] = r;
          ss = fmaf(r, r, ss);
        }
      }
    }
    ss = block_sum_f(ss, red);
    if (tid == 0) part = ss;
  }
  cluster_sync_all();
  if (slot >= 0) {
    float ss = 0.f;
#pragma unroll 1
    for (int i = 0; i < (int)gridDim.x; ++i) ss += ld_cluster_f32(&part, i);
    const float rs = 1.0f / sqrtf(ss / (float)a.vdim + a.eps);
#pragma unroll 1
    for (int j = tid; j < own; j += kStepT) {
      const float z = sgate[j], sig = sigmoid_f(z);
      a.out[(long long)h * a.vdim + c_lo + j] = so[j] * rs * (j == tid ? norm : bf(nw + j)) * (a.gate_kind == kGateSilu ? z * sig : sig);
    }
    // A CTA that starts after this store still finds `pos` in its own slot: only the other slot's tag changes.
    if (rank == 0 && h == 0 && tid == 0) {
      a.tags[1 - slot] = pos + 1;
      if (pos == 0) a.tags[1] = -1;
    }
  }
  if (gridDim.x > 1) cluster_sync_all();                                 // nobody leaves while its sum is read
}

constexpr int kMaxSmem = 220 * 1024;

template <class K>
int allow_smem(K kern, bool& done) {
  if (done) return 0;
  const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxSmem);
  done = e == cudaSuccess;
  return (int)e;
}

template <int KIND, int L, int NV>
int launch_chunk(const StateChunkArgs& a, cudaStream_t stream) {
  static bool configured = false;
  if (const int rc = allow_smem(state_chunk_kernel<KIND, L, NV, false>, configured)) return rc;
  constexpr int PER_WARP = 32 / L * kQuad;
  const int C = a.vdim + extra_columns<KIND>();
  int warps = 8;                               // as few as it takes to give most SMs a CTA
  while (warps > 1 && a.heads * ((C + warps * PER_WARP - 1) / (warps * PER_WARP)) < 100) warps /= 2;
  const int cols = warps * PER_WARP, blocks = (a.rows + kStateBlock - 1) / kStateBlock;
  int pieces = KIND == kStateDelta || blocks < 16 ? 1 : blocks / 8 < kStatePieces ? blocks / 8 : kStatePieces;
  const int per = (blocks + pieces - 1) / pieces;
  pieces = (blocks + per - 1) / per;
  if (KIND == kStateNormalized) {
    if (const int rc = launch_pdl(gate_scan_kernel, dim3(a.heads), dim3(kScanT), 0, stream, false, a)) return rc;
  }
  constexpr int NC = NV * 4 * L / 32 < 2 ? 1 : 2;                        // wider slices cost occupancy
  if (const int rc = launch_pdl(state_blocks_kernel<KIND, NC>, dim3(blocks, (a.heads + 3) / 4), dim3(128), 0, stream, false, a)) return rc;
  const dim3 grid((C + cols - 1) / cols, a.heads, pieces);
  const int smem = 4 * (kStages * (state_record(KIND, a.dim) + kStateBlock * cols) + warps * (32 / L) * 2 * kStateBlock * kQuad);
  if (smem > kMaxSmem) return -7;
  if constexpr (KIND != kStateDelta) {
    if (pieces > 1) {
      static bool sums_configured = false;
      if (const int rc = allow_smem(state_chunk_kernel<KIND, L, NV, true>, sums_configured)) return rc;
      const int rc = launch_pdl(state_chunk_kernel<KIND, L, NV, true>, dim3(grid.x, grid.y, pieces - 1), dim3(warps * 32), smem, stream, false, a, per);
      if (rc) return rc;
    }
  }
  return launch_pdl(state_chunk_kernel<KIND, L, NV, false>, grid, dim3(warps * 32), smem, stream, false, a, per);
}
// L * NV * 4 = state_row(dim).  Fewer lanes per column mean fewer reductions but also fewer warps: the delta rule, which has no pieces
// to spread, takes more lanes.
template <int KIND>
int chunk_by_dim(const StateChunkArgs& a, cudaStream_t stream) {
  if (a.dim <= 32) return launch_chunk<KIND, 8, 1>(a, stream);
  if constexpr (KIND == kStateDelta) {
    if (a.dim <= 64) return launch_chunk<KIND, 16, 1>(a, stream);
    if (a.dim <= 128) return launch_chunk<KIND, 16, 2>(a, stream);
  } else {
    if (a.dim <= 64) return launch_chunk<KIND, 8, 2>(a, stream);
    if (a.dim <= 128) return launch_chunk<KIND, 8, 4>(a, stream);
  }
  if (a.dim <= 256) return launch_chunk<KIND, 16, 4>(a, stream);
  return launch_chunk<KIND, 32, 4>(a, stream);
}
template <int KIND, int NV>
int launch_state_step(const StateStepArgs& a, cudaStream_t stream, bool pdl) {
  static bool configured = false;
  if (const int rc = allow_smem(state_step_kernel<KIND, NV>, configured)) return rc;
  int ctas = 1;                                // per head: a cluster, while that fits the SMs and leaves 16 columns each
  while (ctas < 8 && a.heads * ctas * 2 <= 148 && a.vdim >= 32 * ctas) ctas *= 2;
  const int per = (a.vdim + ctas - 1) / ctas;
  const int base = 4 * step_floats(NV * 4 * kLanes, per, (int)a.decay_ld, (int)a.gate_ld);
  const int weights = 2 * (int)((KIND == kStateNormalized ? 0 : a.dim * a.decay_ld) + (a.gate_w ? per * a.gate_ld : 0));
  const bool staged = base + weights <= kMaxSmem;
  if (base > kMaxSmem) return -7;
  return launch_cluster(state_step_kernel<KIND, NV>, dim3(ctas, a.heads), dim3(kStepT), dim3(ctas, 1, 1), base + (staged ? weights : 0), stream, pdl, a, per, (int)staged);
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
extern "C" int nrt_state_block_floats(int kind, int dim) { return state_record(kind, dim); }       // per (block, head)
extern "C" long long nrt_state_sum_floats(int kind, int heads, int dim, int vdim) {
  return kind == kStateDelta ? 0 : (long long)(kStatePieces - 1) * heads * (vdim + (kind == kStateNormalized) + 1) * pad4(dim);
}
extern "C" int nrt_state_step_args_size() { return (int)sizeof(StateStepArgs); }

extern "C" int nrt_state_chunk(int kind, const void* args, void* stream) {
  StateChunkArgs a;
  memcpy(&a, args, sizeof(a));
  if (a.rows < 1 || !sizes_ok(a.heads, a.kv_heads, a.dim, a.vdim) || a.state_stride % 4 || !a.blocks || (kind != kStateDelta && !a.sums)) return -3;
  if (a.history && (a.hist_rows < 1 || a.hist_rows < 2 * (a.taps - 1))) return -3;
  if ((kind != kStateNormalized && !a.g) || (kind == kStateNormalized && (!a.gi || !a.gf || !a.den || !a.keep)) || (kind == kStateDelta && !a.beta) || (kind == kStateBonus && !a.u)) return -3;
  if (kind == kStateDelta) return chunk_by_dim<kStateDelta>(a, S(stream));
  if (kind == kStateBonus) return chunk_by_dim<kStateBonus>(a, S(stream));
  if (kind == kStateNormalized) return chunk_by_dim<kStateNormalized>(a, S(stream));
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
