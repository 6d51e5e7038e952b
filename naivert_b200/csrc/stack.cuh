// Argument structs and small device helpers of the layer-stack kernels: the mechanisms from which models of
// freely ordered layers (latent and chunked grouped-query attention, gated linear recurrence, matrix-state recurrences,
// dense and expert feed-forwards, norms before and after a sublayer, looped layers) are put together.  Every size and constant is a field; nothing here belongs to one model.
//
// Activation buffers come in two forms: bf16 (`f32` = 0: tensor-core products) and float (`f32` = 1: everything in
// true 32-bit on the CUDA cores).  Weights are bf16 in both.  The residual stream, norms, routers, attention scores,
// recurrent state and recurrence gates are float in both.
#pragma once
#include "ptx.cuh"

#include <float.h>

namespace nrt {

// ------------------------------------------------------------------------------------ chunk (prefill) products
enum StackEpi : int {
  kSEpiStore = 0,      // acc * scale
  kSEpiBias = 1,       // acc + bias; features below `act_cols` go through the tanh form of GELU
  kSEpiTranspose = 2,  // acc stored feature-major: out[feature][token] (bf16)
  kSEpiClampedGlu = 3, // two products g, u: g = min(g, limit), u = clamp(u), g * sigmoid(alpha g) * (u + 1)
  kSEpiSiluGlu = 4,    // two products g, u: silu(g) * u
  kSEpiRelu2 = 5,      // relu(acc)^2
  kSEpiTanh = 6,       // tanh(acc)
  kSEpiDecaySoft = 7,  // exp(-rate * softplus(acc + bias)), rate per feature
  kSEpiDecayExp = 8,   // exp(-exp(acc + bias))
};

struct StackGemmArgs {
  const void* act;              // float form: activations, element (row, z, k) at row * act_ld + z * act_zstride + k
  const __nv_bfloat16* w;       // float form: weights, element (z, n, k) at z * w_zstride + n * w_ld + k
  const __nv_bfloat16* w2;      // second matrix of the two-product epilogues
  long long act_ld, act_zstride, w_ld, w_zstride;
  int n, k, rows;               // features per group, inner size, token rows
  int zcount;                   // independent groups (plain form): heads or blocks with their own weights and columns
  const int* n_items;           // item form (routed experts): number of row segments, else null
  const int* item_z;            // weight group of a segment
  const int* item_row;          // its first row
  int max_items;
  int item_rows;                // rows of a segment
  void* out;
  int out_f32;                  // element type of `out`
  long long out_ld, out_zstride;
  const __nv_bfloat16* bias;    // [zcount][n]
  const float* rate;            // [n] (kSEpiDecaySoft)
  int act_cols;
  float scale, limit, alpha;
  uint32_t* status;
};

// ------------------------------------------------------------------------------------ rows
enum NormKind : int {
  kNormRms = 0,        // x / sqrt(mean(x^2) + eps) * w
  kNormLayer = 1,      // (x - mean) / sqrt(mean((x - mean)^2) + eps) * w
};

struct StackRowArgs {
  // where the stream comes from: an embedding gather (tokens != null), else x as it stands
  const int* tokens;
  const __nv_bfloat16* table;
  int vocab;
  float embed_scale;
  // sublayer output added through its own norm (null: none); with `slot_of` the row is the weighted sum of top_k rows
  const float* y;
  long long y_ld;
  const int* slot_of;           // [rows][top_k]
  const float* probs;           // [rows][top_k]
  int top_k;
  const __nv_bfloat16* post_w;
  // second branch of a sublayer with two mixers (null: none): y becomes the mean of the branches, scaled to unit RMS times join_w / join_w2
  const float* y2;
  const __nv_bfloat16* join_w;
  const __nv_bfloat16* join_w2;
  const __nv_bfloat16* add;     // vector added to the stream afterwards (null: none)
  float* x;                     // [rows][width] in / out
  const __nv_bfloat16* pre_w;   // norm of the next sublayer (null: none)
  int norm;                     // NormKind of post_w and pre_w
  int copy_h;                   // without pre_w: the stream itself is the next sublayer's input
  void* h;
  int h_f32;
  long long h_ld;
  int width, rows;
  float eps;
};

// ------------------------------------------------------------------------------------ latent attention
struct LatentPrepArgs {
  const float* proj;            // [rows][ld]: query latent | key/value latent | output gate (raw)
  long long ld;
  int rows, q_rank, kv_rank;
  const __nv_bfloat16* q_w;
  const __nv_bfloat16* kv_w;
  float eps;
  void* cq;                     // [rows][cq_ld]
  long long cq_ld;
  void* cache;                  // [capacity][cache_ld], row = position
  long long cache_ld;
  int f32;
  const int* pos0;
  int capacity;
};

// Attention of chunk rows over a block of keys.  Query head h uses key / value head h / group.  With `window` > 0 positions are
// cut into chunks of that many ([0, window), [window, 2 window), ...), and a query sees only keys of its own chunk.
struct LatentAttnArgs {
  const void* q;                // [rows][heads * dim]
  const void* k;                // keys of the block [kv_rows][heads / group * dim]
  const void* v;                // simple form: [kv_rows][heads / group * vdim]; tensor-core form: feature-major [heads / group * vdim][v_ld]
  long long v_ld;
  int group;                    // query heads per key / value head
  int window;                   // chunk length of the mask, 0: causal only
  int k_row0;                   // tensor-core form: row of the key map that holds position kv0
  const float* gate;            // raw output gate (null: none), element (row, head * vdim + j) at row * gate_ld + ...
  long long gate_ld;
  void* out;                    // [rows][heads * vdim]
  int f32;
  int rows, heads, dim, vdim;   // storage sizes (padded)
  float scale;
  const int* pos0;              // position of row 0
  int kv0, kv_rows;             // positions covered by k / v
  int first, last;              // first: no carried state; last: normalise, gate and store
  float* state;                 // carried softmax state [rows][heads][vdim + 2] (max, sum, unnormalised output)
  uint32_t* status;
};

struct LatentDecodeArgs {
  const float* q;               // [heads][rank] queries taken into the latent space
  const void* cache;            // [capacity][cache_ld]
  long long cache_ld;
  int f32;
  int heads, rank;
  float scale;
  const int* pos0;
  float* part;                  // [splits][heads][latent_part_row(rank)]: max, sum, -, -, unnormalised latent output
  int splits;
};

// ------------------------------------------------------------------------------------ gated linear recurrence
struct RecurrenceArgs {
  // short convolution
  const void* xy;               // [rows][xy_ld]: gate branch | recurrence branch
  long long xy_ld;
  const __nv_bfloat16* conv;    // [width][taps]
  const __nv_bfloat16* conv_b;
  int taps;
  float* history;               // [hist_rows][width] inputs of earlier positions, slot = position % hist_rows
  int hist_rows;
  void* u;                      // [rows][blocks][block_pad]
  // recurrence
  const float* gates;           // [rows][blocks][2 * block]: pre-activation r | i of every block (scratch: the scan
                                // replaces them by decay and drive)
  const float* softplus_lam;    // [width]
  float decay;                  // log a = -decay * r * softplus(lam)
  float* state;                 // [2][width] state after a position
  int* tags;                    // [2]: number of tokens each state slot has seen
  float* agg;                   // [chunks][2][width] scratch: decay product, local end state
  void* out;                    // [rows][out_ld]
  long long out_ld;
  int f32;
  int rows, width, blocks, block, block_pad;
  const int* pos0;
  uint32_t* status;
};

// ------------------------------------------------------------------------------------ chunked grouped-query attention
// Queries, keys and values of a token as one product left them (biases added); norms per head, rotation of the first
// rot_dims columns (halves paired, angle = position * freq[i]), queries times `scale`.
struct GroupPrepArgs {
  const float* proj;            // [rows][ld]: queries from q_off, keys from k_off, values from v_off
  long long ld;
  int q_off, k_off, v_off;
  int rows, heads, kv_heads, dim, vdim, dp, vp;      // dp, vp: storage widths of a head
  const __nv_bfloat16* q_norm;  // [dim] (null: none)
  const __nv_bfloat16* k_norm;
  const float* freq;            // [rot_dims / 2]
  int rot_dims;
  float eps, scale;
  void* q;                      // [rows][heads * dp]
  void* k_cache;                // [capacity][kv_heads * dp], row = position
  void* v_cache;                // [capacity][kv_heads * vp]
  int f32;
  const int* pos0;
  int capacity;
};

struct TransposeArgs {          // cols and dst_ld even
  const __nv_bfloat16* src;     // [rows][cols]
  __nv_bfloat16* dst;           // [cols][dst_ld]
  long long dst_ld;
  int rows, cols;
};

// One token: preparation as above, then attention over the visible keys, split over a cluster that merges its parts.
struct GroupDecodeArgs {
  GroupPrepArgs p;              // rows = 1; q unused
  int window;                   // chunk length of the mask, 0: causal only
  int splits;                   // cluster size
  float* out;                   // [heads * vdim]
};

// ------------------------------------------------------------------------------------ matrix-state recurrences
// Every head carries a matrix S [dim x vdim] (stored per value column: [vdim][dim4], dim4 = dim rounded up to four).
enum StateKind : int {
  // With S' = diag(g) S ahead of the update, o = q^T S read out:
  kStateDelta = 0,     // S' moves towards v at k by the step beta: S = S' + beta k (v - k^T S')^T; read after the update
  kStateBonus = 1,     // S = S' + k v^T; read before decay and update, plus the token's own term (q . u k) v
  kStateNormalized = 2,// S = a S + b k v^T with scalar a, b from a running maximum; read after; sums of k weighted alike give the normaliser
};
enum GateKind : int { kGateSigmoid = 0, kGateSilu = 1 };

// Chunk rows are worked off in blocks of kStateBlock tokens.  With c_t the product of the block's decays up to token t (per key
// channel), everything the block needs from the state S at its start are products with c_t k_t and c_t q_t, and what is left of the
// tokens' influence on one another are a few numbers per pair.  `blocks` holds a record per (block, head), written by a kernel of its
// own: [c_t k_t (delta only)] [c_t q_t] [k_t times the decays behind it], kStateBlock rows each, then the block's whole decay; rows are
// padded with zeros to state_row(dim).  Then 64 pair coefficients, element [t][s]: s <= t: weight of token s's update in the
// read-out of token t; s > t: what token t's update adds to S^T k at token s (delta).  Then the step sizes (delta).
constexpr int kStateBlock = 8;
constexpr int kStatePieces = 8;      // parts of a chunk that the recurrences without S^T k work off side by side
__host__ __device__ inline int state_row(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : dim <= 256 ? 256 : 512; }
__host__ __device__ inline int state_record(int kind, int dim) {
  return ((kind == kStateDelta ? 3 : 2) * kStateBlock + 1) * state_row(dim) + kStateBlock * kStateBlock + kStateBlock;
}

struct StateChunkArgs {
  const float* q;               // element (row, key head, d) at row * q_ld + key head * dim + d
  const float* k;
  const float* v;               // element (row, head, j) at row * v_ld + head * vdim + j
  const float* g;               // decay per head and key channel (delta, bonus)
  long long q_ld, k_ld, v_ld, g_ld;
  int rows, heads, kv_heads, dim, vdim;
  float q_scale;
  const float* beta;            // delta: raw step size, element (row, head) at row * beta_ld + head
  long long beta_ld;
  const __nv_bfloat16* u;       // bonus: [heads][dim]
  const float* gi;              // normalized: raw input and forget gates, element (row, head) at row * gate_ld + head
  const float* gf;
  long long gate_ld;
  float cap;
  float* keep;                  // normalized, scratch: [rows][heads][2] = factor on the state, factor on the new term
  float* blocks;                // scratch: [blocks][heads][state_record]
  float* sums;                  // bonus, normalized, scratch: [kStatePieces - 1][heads][columns][dim4] states of a piece from zero, then
                                // [kStatePieces - 1][heads][dim4] decays of a piece
  float* o;                     // [rows][heads * vdim]
  float* den;                   // normalized: [rows][heads][2] = n . q, exp(-m)
  float* state;                 // [2][state_stride]: heads x columns x dim4, then (normalized) the running maxima
  long long state_stride;
  int* tags;                    // [2]: number of tokens each state slot has seen
  // inputs of a short convolution whose last rows are kept for the next chunk (null: none)
  const float* hist_src;        // [rows][hist_ld], first hist_cols columns
  long long hist_ld;
  int hist_cols, taps, hist_rows;
  float* history;               // [hist_rows][hist_cols], slot = position % hist_rows
  const int* pos0;
  uint32_t* status;
};

// Short causal convolution + SiLU of the q | k | v columns of a projection; q and k heads become unit vectors (q times q_scale).
// The remaining columns named by `low` are copied to an operand buffer.
struct ShortConvArgs {
  const float* proj;            // [rows][ld]: q [kv_heads * dim] | k [kv_heads * dim] | v [heads * vdim] | ...
  long long ld;
  int rows, heads, kv_heads, dim, vdim, taps;
  const __nv_bfloat16* conv;    // [columns][taps]
  const float* history;         // [hist_rows][columns]
  int hist_rows;
  float q_scale;
  float* q;                     // [rows][kv_heads * dim]
  float* k;
  float* v;                     // [rows][heads * vdim]
  int low_off, low_cols;        // columns copied to `low` [rows][low_ld]
  int low2_off, low2_cols, low2_at;   // and from low2_at on
  void* low;
  long long low_ld;
  int f32;
  const int* pos0;
};

// Mixes of a token with its predecessor: out[row][s] = x + (x_before - x) * mu[s]
struct TokenMixArgs {
  const float* x;               // [rows][width]
  int rows, width, mixes;
  const __nv_bfloat16* mu;      // [mixes][width]
  void* out;                    // [rows][mixes][out_ld]
  long long out_ld;
  int f32;
  float* shift;                 // state slot s keeps the last row at shift + s * state_stride
  long long state_stride;
  const int* tags;
  const int* pos0;
  uint32_t* status;
};

// Read-out of a matrix state: each head divided by its root mean square, times a weight, times a gate.
struct HeadGateArgs {
  const float* o;               // [rows][heads * vdim]
  const float* den;             // [rows][heads][2] (null: none): o is first divided by max(|n . q|, exp(-m)) + 1e-6
  const __nv_bfloat16* norm;    // [vdim] shared (norm_per_head = 0) or [heads * vdim]
  int norm_per_head;
  const float* gate;            // raw, element (row, head * vdim + j) at row * gate_ld + ...
  long long gate_ld;
  int gate_kind;
  void* out;                    // [rows][out_ld]
  long long out_ld;
  int f32, rows, heads, vdim;
  float eps;
};

// One token of a matrix-state mixer: unit vectors, low-rank decay and gate, state update, read-out, head norm and gate.
struct StateStepArgs {
  int kind, heads, kv_heads, dim, vdim;
  const float* proj;            // the token's projections; offsets of its parts
  int q_off, k_off, v_off;
  int unit;                     // q and k become unit vectors
  float q_scale;
  int beta_off;                 // delta
  const __nv_bfloat16* u;       // bonus
  int gi_off, gf_off;           // normalized
  float cap;
  // decay = exp(-rate softplus(z + bias)) (rate != null) or exp(-exp(z + bias)), z = decay_w act(in)
  int low_off, low_rank, low_tanh;
  const __nv_bfloat16* decay_w; // [heads * dim][decay_ld]
  long long decay_ld;
  const __nv_bfloat16* decay_b; // [heads * dim]
  const float* rate;            // [heads * dim]
  // gate: raw columns of the projection, or low-rank (gate_w != null)
  int gate_off, gate_rank, gate_kind;
  const __nv_bfloat16* gate_w;  // [heads * vdim][gate_ld]
  long long gate_ld;
  const __nv_bfloat16* norm;
  int norm_per_head;
  float eps;
  float* state;
  long long state_stride;
  int* tags;
  float* out;                   // [heads * vdim]
  const int* pos0;
  uint32_t* status;
};

struct MoeGatherArgs {
  const void* h;                // [rows][h_ld]
  long long h_ld;
  void* sorted;                 // [cap][h_ld]
  const int* slot_of;           // [rows][top_k]
  int rows, top_k, row_bytes;   // bytes of a row to copy (a multiple of 16)
  int cap;
};

// ------------------------------------------------------------------------------------ one-token step
enum StepPro : int {
  kProResidual = 0,    // stream update + norm: x_out = x + rms(y) * post_w + add; input = rms(x_out) * in_w
  kProNorm = 1,        // input = rms(in) * in_w
  kProLoad = 2,        // input = in + group * in_gstride
  kProMerge = 3,       // input = softmax-merged latent output of head `group` from the attention partials
  kProMix = 5,         // stream update, then input of group g = x_out + (x_before - x_out) * mu[g] (x_before: the previous token's)
  kProExperts = 4,     // inputs of the chosen experts side by side, each times its weight: out = sum_j W[ids[j]] (p[j] in[j])
};
enum StepEpi : int {
  kTEpiStore = 0,      // acc * scale (+ bias); rows from `sig_from` on through a sigmoid
  kTEpiConv = 1,       // + bias; rows < width: GELU (tanh form); others: convolution input -> u, history
  kTEpiGate = 2,       // acc * gate[row]
  kTEpiGlu = 3,        // two products: clamped GLU (glu_kind 0) or SiLU GLU (1)
  kTEpiRecur = 4,      // two products (r, i) + biases: recurrence step, times the gate branch
  kTEpiConvSilu = 5,   // rows < conv_rows: short convolution without a bias, SiLU; others: stored
  kTEpiRelu2 = 6,      // relu(acc)^2
};

struct StepArgs {
  // input
  const int* tokens;
  const __nv_bfloat16* table;
  int vocab;
  float embed_scale;
  const float* x;
  const float* y;
  const __nv_bfloat16* post_w;
  const float* y2;              // second half of a sublayer of two mixers (StackRowArgs)
  const __nv_bfloat16* join_w;
  const __nv_bfloat16* join_w2;
  int norm;                     // NormKind of post_w and in_w (stream prologues)
  int raw_in;                   // the stream itself is the input (no in_w)
  const __nv_bfloat16* mu;      // kProMix: [groups][k]
  float* shift;                 // kProMix: the previous token's stream, state slot s at shift + s * state_stride
  long long state_stride;
  const __nv_bfloat16* add;
  float* x_out;
  const float* in_;
  long long in_gstride;
  const __nv_bfloat16* in_w;
  float eps;
  int k;
  // attention partials
  const float* part;
  int splits;
  // weights
  const __nv_bfloat16* w;
  const __nv_bfloat16* w2;
  long long w_ld, w_gstride, w2_gstride;
  int groups, n;                // groups x n output rows
  int n_last;                   // rows of the last group (0: n)
  int conv_rows;                // kTEpiConvSilu
  int segs;                     // chosen experts whose products are summed (kProExperts), else 1
  const int* ids;               // [segs] their weight groups
  const float* probs;           // [segs] their weights
  // output
  float* out;                   // [groups][n]
  float scale;
  int sig_from;
  const __nv_bfloat16* bias;
  const __nv_bfloat16* bias2;
  const float* gate;
  int glu_kind;
  float limit, alpha;
  // latent key/value row appended by this launch (kProNorm of the query latent)
  const float* lat_in;
  const __nv_bfloat16* lat_w;
  int lat_rank;
  void* lat_cache;
  long long lat_ld;
  int f32;                      // caches and rounding of the float form
  // recurrence
  const __nv_bfloat16* conv;
  const __nv_bfloat16* conv_b;
  int taps;
  float* history;
  int hist_rows;
  float* u;
  const float* softplus_lam;
  float decay;
  float* state;
  int* tags;
  const int* pos0;
  int capacity;
  uint32_t* status;
};

// Context splits of the one-token attention: rows per split (a multiple of the kernels' 64-row tile) and the layout of a
// partial result.
constexpr int kMaxSplits = 256;
__host__ __device__ inline int latent_split_rows(int n, int splits) { return ((n + splits - 1) / splits + 63) / 64 * 64; }
__host__ __device__ inline int latent_part_row(int rank) { return (rank + 3) / 4 * 4 + 4; }

// ------------------------------------------------------------------------------------ math
__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float gelu_tanh_f(float z) {
  return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
__device__ __forceinline__ float clamped_glu(float g, float u, float limit, float alpha) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g * sigmoid_f(alpha * g) * (u + 1.0f);
}
__device__ __forceinline__ float silu_glu(float g, float u) { return g * sigmoid_f(g) * u; }
__device__ __forceinline__ float silu_f(float z) { return z * sigmoid_f(z); }
__device__ __forceinline__ float relu2_f(float z) { z = fmaxf(z, 0.f); return z * z; }
// log(1 + t) for 0 <= t <= 1: twice the area tangent of s = t / (2 + t) <= 1/3, as its power series (the next term is below 2e-8)
__device__ __forceinline__ float log1p_unit(float t) {
  const float s = __fdividef(t, 2.0f + t), q = s * s;
  float p = fmaf(q, 1.0f / 13.0f, 1.0f / 11.0f);
  p = fmaf(q, p, 1.0f / 9.0f);
  p = fmaf(q, p, 1.0f / 7.0f);
  p = fmaf(q, p, 1.0f / 5.0f);
  p = fmaf(q, p, 1.0f / 3.0f);
  p = fmaf(q, p, 1.0f);
  return 2.0f * s * p;
}
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1p_unit(expf(-fabsf(z))); }
__device__ __forceinline__ float soft_cap(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float decay_soft(float z, float rate) { return expf(-rate * softplus_f(z)); }
__device__ __forceinline__ float decay_exp(float z) { return expf(-expf(z)); }

__device__ __forceinline__ float lane_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
// Sum over the block (blockDim a multiple of 32, at most 1024); every thread gets it.  `red`: 33 floats of shared memory.
__device__ __forceinline__ float block_sum_f(float v, float* red) {
  v = lane_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float s = 0.f;
#pragma unroll 1
  for (int i = 0; i < nw; ++i) s += red[i];
  return s;
}
__device__ __forceinline__ float bf(const __nv_bfloat16* p) { return __bfloat162float(*p); }

__device__ __forceinline__ void store_act(void* base, long long i, float v, int f32) {
  if (f32) reinterpret_cast<float*>(base)[i] = v;
  else reinterpret_cast<__nv_bfloat16*>(base)[i] = __float2bfloat16_rn(v);
}
__device__ __forceinline__ float load_act(const void* base, long long i, int f32) {
  return f32 ? reinterpret_cast<const float*>(base)[i] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(base)[i]);
}

// State slot that holds the recurrence after `pos` tokens; -1: none (recorded as a broken hand-over).  Position 0
// starts from zero and writes slot 0.
__device__ __forceinline__ int state_slot(const int* tags, int pos, uint32_t* status) {
  if (pos == 0) return 1;
  const int t0 = *reinterpret_cast<const volatile int*>(tags), t1 = *reinterpret_cast<const volatile int*>(tags + 1);
  if (t0 == pos) return 0;
  if (t1 == pos) return 1;
  report(status, kSiteState);
  return -1;
}

}  // namespace nrt
