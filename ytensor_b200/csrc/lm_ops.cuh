// Mechanisms of the language models that are not part of the reference's operator set, each with its constants as
// parameters so that any model can be put together from them: linear layers with fused activations and grouped
// (mixture-of-experts) products, norms around a sublayer, attention over a sliding window with capped scores and a
// K/V ring, values mixed with those of an earlier layer, attention over a cache of latents with a rotated key shared by
// the heads, linear attention with a decayed state, output gates, softmax and sigmoid routers with a choice correction,
// expert groups and identity experts, and the single-token forms of all of them (csrc/lm_decode.cu).
#pragma once
#include "ytc_common.cuh"

namespace ytk {

// ---------------------------------------------------------------- scalar helpers
#ifdef __CUDACC__
__device__ __forceinline__ uint16_t bf16_rn_bits(float x) {  // round to nearest even
  const __nv_bfloat16 h = __float2bfloat16_rn(x);
  return *reinterpret_cast<const uint16_t*>(&h);
}
__device__ __forceinline__ uint32_t pack_bf16x2_rn(float lo, float hi) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&h);
}
__device__ __forceinline__ float lm_gelu_erf(float z) { return 0.5f * z * (1.f + erff(z * 0.70710678118654752f)); }
__device__ __forceinline__ float lm_silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float lm_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float lm_relu2(float z) {
  z = fmaxf(z, 0.f);
  return z * z;
}
// Gate bounded above, linear part bounded on both sides: g sigmoid(alpha g) (u + shift).
__device__ __forceinline__ float lm_clamped_gate(float gate, float up, float limit, float alpha, float shift) {
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return g / (1.f + expf(-alpha * g)) * (u + shift);
}
__device__ __forceinline__ float lm_sigmoid_fast(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }
__device__ __forceinline__ float lm_silu_fast(float z) { return __fdividef(z, 1.f + __expf(-z)); }  // bf16 results

// Activations and caches are stored as float or as bf16 bits: 8 elements at a time.
template <typename T>
struct Vec8;
template <>
struct Vec8<float> {
  static __device__ __forceinline__ void load(const float* p, float (&f)[8]) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
    f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
  }
  static __device__ __forceinline__ void store(float* p, const float (&f)[8]) {
    reinterpret_cast<float4*>(p)[0] = make_float4(f[0], f[1], f[2], f[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(f[4], f[5], f[6], f[7]);
  }
};
template <>
struct Vec8<uint16_t> {
  static __device__ __forceinline__ void unpack(const uint4& w, float (&f)[8]) {
    const uint32_t u[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      f[2 * i] = __uint_as_float(u[i] << 16);
      f[2 * i + 1] = __uint_as_float(u[i] & 0xFFFF0000u);
    }
  }
  static __device__ __forceinline__ void load(const uint16_t* p, float (&f)[8]) {
    unpack(*reinterpret_cast<const uint4*>(p), f);
  }
  static __device__ __forceinline__ void store(uint16_t* p, const float (&f)[8]) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2_rn(f[0], f[1]), pack_bf16x2_rn(f[2], f[3]),
                                              pack_bf16x2_rn(f[4], f[5]), pack_bf16x2_rn(f[6], f[7]));
  }
};
#endif

// ---------------------------------------------------------------- linear layers
// What happens to a product before it is stored. EPI_NONE: as ytcuda_gemm stores it; EPI_BF16: bf16, nearest even;
// EPI_GELU_ERF: exact (erf) gelu; EPI_SWIGLU_PAIRS: the weight rows alternate gate_j, up_j and silu(gate_j) * up_j is
// stored at column j, half as many columns as weight rows; EPI_RELU2: max(z, 0)^2; EPI_SILU: silu in the first act_cols
// columns, the others as they are; EPI_CLAMP_PAIRS: gate and up rows as in EPI_SWIGLU_PAIRS, g = min(gate, limit),
// u = up bounded to [-limit, limit], g sigmoid(alpha g) (u + shift). All but EPI_NONE store bf16 (linear_tc) or fp32
// (linear_f32).
enum { EPI_NONE = 0, EPI_BF16 = 1, EPI_GELU_ERF = 2, EPI_SWIGLU_PAIRS = 3, EPI_RELU2 = 4, EPI_SILU = 5, EPI_CLAMP_PAIRS = 6 };
inline bool epi_pairs(int epi) { return epi == EPI_SWIGLU_PAIRS || epi == EPI_CLAMP_PAIRS; }
struct LinearEpilogue {
  int epi = EPI_NONE;
  int act_cols = 0;
  float limit = 0.f, alpha = 1.702f, shift = 1.f;
  // grouped product: 128-row block i of x is multiplied by rows tile_group[i] * n .. of the stacked weight (`groups`
  // matrices of n rows), blocks with tile_group[i] < 0 are passed over
  const int* tile_group = nullptr;
  int groups = 1;
};
#ifdef __CUDACC__
// The fp32 forms: column n of a plain epilogue, a (gate, up) pair of a gated one.
__device__ __forceinline__ float lm_activation(const LinearEpilogue& ex, float z, int n) {
  if (ex.epi == EPI_GELU_ERF) return lm_gelu_erf(z);
  if (ex.epi == EPI_RELU2) return lm_relu2(z);
  if (ex.epi == EPI_SILU && n < ex.act_cols) return lm_silu(z);
  return z;
}
__device__ __forceinline__ float lm_gated(const LinearEpilogue& ex, float gate, float up) {
  return ex.epi == EPI_CLAMP_PAIRS ? lm_clamped_gate(gate, up, ex.limit, ex.alpha, ex.shift) : lm_silu(gate) * up;
}
#endif
constexpr int LM_GROUP_ROWS = 128;
// y[m, n] = epilogue(x[m, k] . W[n, k]^T): x bf16, on the tensor cores (csrc/gemm.cu).
int linear_tc(const void* x, int64_t ldx, const void* w, int64_t ldw, void* y, int64_t ldy, int out_dtype, int m, int n,
              int k, const LinearEpilogue& ex, cudaStream_t st);
// The same with fp32 x and y and fp32 products (csrc/lm_rows.cu).
int linear_f32(const float* x, int64_t ldx, const uint16_t* w, int64_t ldw, float* y, int64_t ldy, int m, int n, int k,
               const LinearEpilogue& ex, cudaStream_t st);

// ---------------------------------------------------------------- residual stream
// x[row] = scale * embedding of ids[row]
int embed_rows(const uint16_t* table, const int* ids, float* x, int64_t rows, int width, int vocab, float scale,
               cudaStream_t st);
// One row of the residual stream per CTA:
//   y    = sublayer output: `y` [rows][ld] fp32, or the weighted sum of the token's experts (slot .. top), or both added
//   x   += y / rms(y) * w_post                      (skipped when w_post is null)
//   h    = x / rms(x) * w_pre -> fp32 or bf16       (w_pre null: h = x; skipped when h is null)
// Rows are `ld` floats (a multiple of 8), the channels past `width` are zero and stay zero.
struct ResidualNorm {
  float* x = nullptr;
  const float* y = nullptr;
  const void* expert_out = nullptr;  // [grouped rows][ld], activation dtype
  const int* slot = nullptr;         // [rows][top]: row of expert_out, -1: the sublayer's input h_in itself, -2: nothing
  const float* weight = nullptr;     // [rows][top], null: all 1
  const void* h_in = nullptr;        // [rows][ld], activation dtype
  int top = 0;
  const float *w_post = nullptr, *w_pre = nullptr;
  void* h = nullptr;
  int dtype = YTC_F32;               // of h, h_in and expert_out
  const int* row_index = nullptr;    // h row i comes from x row row_index[i] (null: i)
  int64_t rows = 0;
  int width = 0, ld = 0;
  float eps = 0.f;
};
int residual_norm(const ResidualNorm& a, cudaStream_t st);

// ---------------------------------------------------------------- attention over a window
// q_len queries at positions pos0 .. per sequence over a K/V ring: position p lies in ring row p % ring. A query sees
// the last `window` positions up to itself (0: all). score = scale * q . k, then softcap * tanh(score / softcap) when
// softcap > 0. Strides are {batch, head, row} in elements. bf16 with head_dim == value_dim in {64, 128} and a ring of
// whole 128-row tiles runs on tcgen05, everything else on the one-warp-per-row kernel (csrc/flash_attn.cu).
struct WindowAttn {
  int dtype = YTC_F32;
  const void *q = nullptr, *k = nullptr, *v = nullptr;
  void* o = nullptr;
  int batch = 1, kv_heads = 1, groups = 1, q_len = 1, head_dim = 0, value_dim = 0;
  int64_t q_st[3] = {}, k_st[3] = {}, v_st[3] = {}, o_st[3] = {};
  int64_t pos0 = 0;
  int window = 0, ring = 0;
  float scale = 1.f, softcap = 0.f;
};
int window_attention(const WindowAttn& a, cudaStream_t st);

// Appends the keys and values of a fused projection to the rings, mixing the values with an earlier layer's:
// v <- (1 - lambda) v + lambda v_first. mix: 0 plain, 1 this layer's values become v_first, 2 mix (csrc/lm_rows.cu).
enum { VMIX_NONE = 0, VMIX_FIRST = 1, VMIX_MIX = 2 };
struct AppendKv {
  int dtype = YTC_F32;
  const void* qkv = nullptr;  // [batch * len][ld]
  int64_t ld = 0;
  int k_off = 0, v_off = 0;   // columns of the first key / value head
  void *k = nullptr, *v = nullptr;  // [batch][kv_heads][ring][dim]
  void* v_first = nullptr;    // [batch * len][kv_heads * vdim]
  const float* lambda = nullptr;
  int mix = VMIX_NONE;
  int batch = 1, len = 1, kv_heads = 1, dim = 0, vdim = 0, ring = 0;
  int64_t pos0 = 0;
};
int append_kv(const AppendKv& a, cudaStream_t st);

// ---------------------------------------------------------------- output gate
// out = norm(in) * w (w null: in) * sigmoid(gate), row by row; in == out is allowed (csrc/lm_rows.cu). The norm runs over
// `width` true channels of the `cols` stored ones (the others are zero).
struct GatedRows {
  int dtype = YTC_F32;
  const void *in = nullptr, *gate = nullptr;
  void* out = nullptr;
  int64_t ld_in = 0, ld_gate = 0, ld_out = 0, rows = 0;
  int cols = 0, width = 0;
  const float* w = nullptr;
  float eps = 0.f;
};
int gated_rows(const GatedRows& a, cudaStream_t st);

// ---------------------------------------------------------------- attention over cached latents
// Every position caches a latent c [rank] (normed) and one rotated key part r [rot], shared by all heads; a row of the
// cache is [c, r]. Per head, key = [Wk c, r] and value = Wv c. Two ways to the same result (csrc/latent_attn.cu):
// many queries expand the cache with one product (row . [Wk | I; Wv]^T) and run window_attention over it; few queries
// move Wk to the query (q Wk, one vector of `rank` per head) and Wv behind the sum, and read the cache as it is.
// Rotation: dimensions 2 i and 2 i + 1 of a vector of `rot` turn by position * base^(-2 i / rot_dims), i < rot_dims / 2.
struct LatentShape {
  int heads = 0, dim = 0, rot = 0, vdim = 0;  // stored sizes, multiples of 8 (rot: of 16)
  int head_ld = 0;                            // elements per query head, >= dim + rot
  int rank = 0;                               // multiple of 16
  int rot_dims = 0;                           // rotated dimensions, the rest of `rot` passes unchanged
  const float* freq = nullptr;                // [rot_dims / 2] base^(-2 i / rot_dims)
  __host__ __device__ int row() const { return rank + rot; }  // cache row
};
// Norms the latent of every row, rotates its key part and stores both into the cache [batch][cap][rank + rot] at
// positions pos0 ..; norms the query latent into cq.
struct LatentAppend {
  int dtype = YTC_F32;
  LatentShape s;
  const void* in = nullptr;   // [batch * len][ld]: columns dq_off .. (q_rank) and dkv_off .. (rank, rot)
  int64_t ld = 0;
  int dq_off = 0, dkv_off = 0, q_rank = 0, q_width = 0, c_width = 0;  // stored query rank, true widths of the norms
  const float *w_q = nullptr, *w_c = nullptr;
  float eps = 0.f;
  void* cq = nullptr;         // [batch * len][q_rank]
  void* cache = nullptr;
  int64_t cap = 0;
  int batch = 1, len = 1;
  int64_t pos0 = 0;
  const int* pos = nullptr;   // decode step: position word (pos0 is ignored)
};
int latent_append(const LatentAppend& a, cudaStream_t st);
// Rotates the `rot` dimensions (from `dim` on) of every head of q [batch * len][heads * head_ld] in place.
int rotate_queries(void* q, int dtype, const LatentShape& s, int batch, int len, int64_t pos0, cudaStream_t st);
// Few query rows: absorbed queries -> partial sums over slices of the cache -> merged and multiplied by Wv.
struct LatentDecode {
  int dtype = YTC_F32;          // of the cache
  int io_dtype = YTC_F32;       // of q and out
  LatentShape s;
  const void* q = nullptr;      // [rows][heads * head_ld], not rotated
  const uint16_t *uk = nullptr, *uv = nullptr;  // [heads * dim][rank], [heads * vdim][rank]
  const void* cache = nullptr;  // [batch][cap][rank + rot]
  int64_t cap = 0;
  int batch = 1, len = 1;       // rows = batch * len
  int64_t pos0 = 0;
  const int* pos = nullptr;     // decode step: position word of the one row (pos0 is ignored)
  int64_t max_keys = 0;         // most keys a query can see (sizes the launch)
  float scale = 1.f;
  float* qa = nullptr;          // [rows][heads][rank + rot]
  float* part = nullptr;        // [rows][heads][splits][rank + 2]: sum, maximum, weight (latent_part_floats)
  void* out = nullptr;          // [rows][heads * vdim]
  int64_t ld_out = 0;
  const LatentAppend* append = nullptr;  // decode step: the new row joins the cache in the first kernel
};
constexpr int LATENT_MAX_ROWS = 16;  // above: expand
int64_t latent_part_floats(const LatentShape& s, int64_t rows, int64_t max_keys);
int latent_decode(const LatentDecode& a, cudaStream_t st);

// ---------------------------------------------------------------- linear attention with a decayed state
// Per head S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t; S [batch][heads][dim][vdim] fp32, carried from call to call.
// bf16 with dim == vdim == 128 and more than a few tokens runs in chunks of 128 on tcgen05, everything else token by
// token on the FMA pipe (csrc/decayed_attn.cu).
struct DecayedAttn {
  int dtype = YTC_F32;
  const void *q = nullptr, *k = nullptr, *v = nullptr;  // head h at column h * dim / h * vdim, row stride ld
  int64_t ld = 0;
  void* o = nullptr;            // [batch * len][ld_o], head h at column h * vdim
  int64_t ld_o = 0;
  float* state = nullptr;
  const float* decay = nullptr; // [heads], device
  int batch = 1, len = 1, heads = 0, dim = 0, vdim = 0;
  bool first = false;           // the state is zero
  const int* pos = nullptr;     // decode step: position word, 0 at a sequence's first token (`first` is ignored)
  int path = 0;                 // 0: automatic, 1: token by token, 2: chunks (an error where the sizes do not allow them)
};
int decayed_attention(const DecayedAttn& a, cudaStream_t st);

// ---------------------------------------------------------------- mixture of experts
// `experts` experts and `identity` pass-through experts share one router: s = softmax(logits), or sigmoid of every logit,
// decides the weights, s + correction the selection (without a correction the logits, which have the order of the scores
// also where these round to the same number). The routes are split into `count` contiguous blocks of one
// size, ranked by their maximal selection score; the `top` routes are taken from the `keep` leading blocks.
enum { ROUTE_SOFTMAX = 0, ROUTE_SIGMOID = 1 };
struct RouterSpec {
  int experts = 0, identity = 0, top = 0, count = 1, keep = 1, score = ROUTE_SOFTMAX;
};
constexpr int LM_MAX_ROUTES = 1024;  // experts + identity
constexpr int LM_MAX_TOP = 32;
// Routes rows of fp32 logits [rows][ld]: choice [rows][top] (router outputs, -1: none), weight [rows][top], rank
// [rows][top] = how many earlier arrivals the expert had, count [experts] += arrivals (csrc/moe.cu).
int moe_route(const float* logits, int64_t ld, const float* correction, int64_t rows, const RouterSpec& r, int* choice,
              float* weight, int* rank, int* count, cudaStream_t st);
// Copies the rows of h [rows][ld] of every chosen expert into blocks of 128 rows per expert: grouped [max rows][ld],
// slot [rows][top] (as in ResidualNorm), tile_group [max rows / 128] (the expert of a block or -1). With `weight` a copy is
// the fp32 row of x times its weight, rounded once.
struct MoeGather {
  const void* h = nullptr;
  const float *x = nullptr, *weight = nullptr;
  int dtype = YTC_F32, ld = 0;
  int64_t rows = 0;
  RouterSpec r;
  const int *choice = nullptr, *rank = nullptr, *count = nullptr;
  void* grouped = nullptr;
  int *slot = nullptr, *tile_group = nullptr;
  int n_tiles = 0;
};
int moe_gather(const MoeGather& g, cudaStream_t st);
inline int moe_max_tiles(int64_t rows, const RouterSpec& r) {
  // every expert with a token may leave one block partly empty
  const int64_t used = rows * r.top < r.experts ? rows * r.top : r.experts;
  return static_cast<int>((rows * r.top) / LM_GROUP_ROWS + used);
}

#ifdef __CUDACC__
// Floats as unsigned integers in the same order; minus infinity is above 0.
__device__ __forceinline__ uint32_t ordered_key(float f) {
  const uint32_t u = __float_as_uint(f);
  return (u & 0x80000000u) ? ~u : (u | 0x80000000u);
}
// One warp takes the largest of its keys (VPL per lane, number j * 32 + lane; equal keys: the lowest number) and
// removes it. False when only keys up to `floor` are left.
template <int VPL>
__device__ __forceinline__ bool warp_take_largest(uint32_t (&key)[VPL], int lane, uint32_t floor, int& index) {
  uint32_t best = 0;
  int bj = 0;
#pragma unroll
  for (int j = 0; j < VPL; ++j)
    if (key[j] > best) {
      best = key[j];
      bj = j;
    }
  const uint32_t top = __reduce_max_sync(0xffffffffu, best);
  if (top <= floor) return false;
  index = static_cast<int>(__reduce_min_sync(0xffffffffu, best == top ? static_cast<uint32_t>(bj * 32 + lane) : 0xffffffffu));
#pragma unroll
  for (int j = 0; j < VPL; ++j)
    if (j * 32 + lane == index) key[j] = 0;
  return true;
}

// One warp routes one token. s: logits of the token in shared memory (overwritten by the scores), c: as many floats of
// scratch; at most 32 * VPL routes. Afterwards lane k < top holds the k-th choice (-1: none) and its weight.
template <int VPL>
__device__ __forceinline__ void warp_route(float* s, float* c, const float* correction, const RouterSpec& r, int lane,
                                           int& choice, float& weight) {
  const int n = r.experts + r.identity;
  const uint32_t floor = ordered_key(-INFINITY);
  float v[VPL], z[VPL];
  float m = -INFINITY;
#pragma unroll
  for (int j = 0; j < VPL; ++j) {
    const int i = j * 32 + lane;
    v[j] = z[j] = i < n ? s[i] : -INFINITY;
    m = fmaxf(m, v[j]);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
  float sum = 0.f;
  if (r.score == ROUTE_SIGMOID) {
    sum = 1.f;
#pragma unroll
    for (int j = 0; j < VPL; ++j) v[j] = j * 32 + lane < n ? lm_sigmoid(v[j]) : 0.f;
  } else {
#pragma unroll
    for (int j = 0; j < VPL; ++j) {
      v[j] = j * 32 + lane < n ? expf(v[j] - m) : 0.f;
      sum += v[j];
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
  }
  uint32_t key[VPL];
#pragma unroll
  for (int j = 0; j < VPL; ++j) {
    const int i = j * 32 + lane;
    key[j] = 0;
    if (i < n) {
      const float p = v[j] / sum, choice_score = correction ? p + correction[i] : z[j];
      s[i] = p;
      c[i] = choice_score;
      key[j] = ordered_key(choice_score);
    }
  }
  __syncwarp();
  if (r.keep < r.count) {
    const int per = n / r.count;
    uint32_t gkey[VPL];
#pragma unroll
    for (int j = 0; j < VPL; ++j) {
      const int g = j * 32 + lane;
      float b = -INFINITY;
      if (g < r.count)
        for (int i = 0; i < per; ++i) b = fmaxf(b, c[g * per + i]);
      gkey[j] = g < r.count ? ordered_key(b) : 0;
    }
    __syncwarp();
#pragma unroll
    for (int j = 0; j < VPL; ++j)
      if (j * 32 + lane < r.count) c[j * 32 + lane] = 0.f;  // from here on: 1 marks a kept group
    __syncwarp();
    for (int k = 0; k < r.keep; ++k) {
      int g = 0;
      if (!warp_take_largest<VPL>(gkey, lane, 0, g)) break;
      if (lane == 0) c[g] = 1.f;
    }
    __syncwarp();
#pragma unroll
    for (int j = 0; j < VPL; ++j) {
      const int i = j * 32 + lane;
      if (i < n && c[i / per] == 0.f) key[j] = floor;
    }
  }
  choice = -1;
  weight = 0.f;
  for (int k = 0; k < r.top; ++k) {
    int i = 0;
    if (!warp_take_largest<VPL>(key, lane, floor, i)) break;
    if (lane == k) {
      choice = i;
      weight = s[i];
    }
  }
}
#endif

// ---------------------------------------------------------------- one new token (csrc/lm_decode.cu)
// Kernels of a decode step, queued as programmatic dependent launches inside a CUDA graph. Activations are fp32
// vectors. The position of the token is read from device memory, so that the graph is the same for every step.
enum { DECODE_EMBED = 0, DECODE_RESIDUAL = 1, DECODE_PLAIN = 2, DECODE_GATED = 3 };
struct DecodeInput {  // how a kernel obtains the vector it multiplies by, in every CTA
  // DECODE_EMBED: x = scale * embedding of *id; DECODE_RESIDUAL: x = x_in + norm(y) * w_post; then, for both,
  // h = norm(x) * w_pre (w_pre null: h = x). DECODE_PLAIN: h = plain. DECODE_GATED: h = norm(plain) * w_pre (w_pre null:
  // plain), times sigmoid(gate) where there is a gate.
  int kind = 2;
  const int* id = nullptr;
  const uint16_t* embed = nullptr;
  int vocab = 0;
  float embed_scale = 1.f;
  const float *x_in = nullptr, *y = nullptr, *w_post = nullptr, *w_pre = nullptr;
  float* x_out = nullptr;   // the new residual row (written by one CTA; another buffer than x_in)
  const float *plain = nullptr, *gate = nullptr;
  int width = 0;            // channels the norms run over
  float eps = 0.f;
};
struct DecodeLinear {
  DecodeInput in;
  const uint16_t* w = nullptr;  // bf16 [n][k]
  int n = 0, k = 0;
  LinearEpilogue ex;            // EPI_NONE, EPI_GELU_ERF, EPI_RELU2 or EPI_SILU
  float* out = nullptr;
  int* advance = nullptr;       // position word to add one to (the last kernel of a step)
};
int decode_linear(const DecodeLinear& a, cudaStream_t st);

struct DecodeAttn {
  int dtype = YTC_F32;          // of the rings
  const float* qkv = nullptr;   // [q heads; k heads; v heads]
  void *k = nullptr, *v = nullptr;
  float* v_first = nullptr;     // [kv_heads * vdim]
  const float* lambda = nullptr;
  int mix = VMIX_NONE;
  float* out = nullptr;         // [heads * vdim]
  const int* pos = nullptr;
  int kv_heads = 1, groups = 1, dim = 0, vdim = 0, ring = 0, window = 0;
  int64_t max_keys = 0;         // most keys a query can see (sizes the launch)
  float scale = 1.f, softcap = 0.f;
};
int decode_attention(const DecodeAttn& a, cudaStream_t st);

struct DecodeRoute {
  DecodeInput in;
  const uint16_t* w = nullptr;  // router [experts + identity][k]
  const float* correction = nullptr;
  int k = 0;
  RouterSpec r;
  float* h = nullptr;           // the normed vector, for the experts
  int* choice = nullptr;        // [top]
  float* weight = nullptr;      // [top]
};
int decode_route(const DecodeRoute& a, cudaStream_t st);

struct DecodeExperts {
  const uint16_t *gate_up = nullptr, *down = nullptr;  // [experts][2 ff][k] (gate_j, up_j alternating), [experts][k][ff]
  int k = 0, ff = 0;
  RouterSpec r;
  LinearEpilogue act;           // EPI_SWIGLU_PAIRS or EPI_CLAMP_PAIRS
  bool scale_input = false;     // a route's weight multiplies the expert's input, not its output
  const uint16_t *shared_gate_up = nullptr, *shared_down = nullptr;  // the shared expert, shared_ff = 0: none
  int shared_ff = 0;
  LinearEpilogue shared_act;
  const int* choice = nullptr;
  const float* weight = nullptr;
  const float* h = nullptr;     // [k]
  float* mid = nullptr;         // [top][ff], then [shared_ff]
  float* out = nullptr;         // [k]
};
int decode_experts(const DecodeExperts& a, cudaStream_t st);

}  // namespace ytk
