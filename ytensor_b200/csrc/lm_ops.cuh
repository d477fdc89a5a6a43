// Mechanisms of the language models that are not part of the reference's operator set, each with its constants as
// parameters so that any model can be put together from them: linear layers with fused activations and grouped
// (mixture-of-experts) products, norms around a sublayer, attention over a sliding window with capped scores and a
// K/V ring, values mixed with those of an earlier layer, a softmax router with a choice correction, expert groups and
// identity experts, and the single-token forms of all of them (csrc/lm_decode.cu).
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
// stored at column j, half as many columns as weight rows. The last three store bf16 (linear_tc) or fp32 (linear_f32).
enum { EPI_NONE = 0, EPI_BF16 = 1, EPI_GELU_ERF = 2, EPI_SWIGLU_PAIRS = 3 };
struct LinearEpilogue {
  int epi = EPI_NONE;
  // grouped product: 128-row block i of x is multiplied by rows tile_group[i] * n .. of the stacked weight (`groups`
  // matrices of n rows), blocks with tile_group[i] < 0 are passed over
  const int* tile_group = nullptr;
  int groups = 1;
};
constexpr int LM_GROUP_ROWS = 128;
// y[m, n] = epilogue(x[m, k] . W[n, k]^T): x bf16, on the tensor cores (csrc/gemm.cu).
int linear_tc(const void* x, int64_t ldx, const void* w, int64_t ldw, void* y, int64_t ldy, int out_dtype, int m, int n,
              int k, const LinearEpilogue& ex, cudaStream_t st);
// The same with fp32 x and y and fp32 products (csrc/lm_rows.cu).
int linear_f32(const float* x, int64_t ldx, const uint16_t* w, int64_t ldw, float* y, int64_t ldy, int m, int n, int k,
               const LinearEpilogue& ex, cudaStream_t st);

// ---------------------------------------------------------------- residual stream
// One row of the residual stream per CTA:
//   y    = sublayer output: `y` [rows][ld] fp32, or the weighted sum of the token's experts (see MoeBuffers)
//   x   += y / rms(y) * w_post                      (skipped without a sublayer output)
//   h    = x / rms(x) * w_pre -> fp32 or bf16       (skipped when w_pre is null)
// Rows are `ld` floats (a multiple of 8), the channels past `width` are zero and stay zero.
struct ResidualNorm {
  float* x = nullptr;
  const float* y = nullptr;
  const void* expert_out = nullptr;  // [grouped rows][ld], activation dtype
  const int* slot = nullptr;         // [rows][top]: row of expert_out, -1: the sublayer's input h_in itself, -2: nothing
  const float* weight = nullptr;     // [rows][top]
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

// ---------------------------------------------------------------- mixture of experts
// `experts` experts and `identity` pass-through experts share one router: s = softmax(logits) decides the weights,
// s + correction the selection. The routes are split into `count` contiguous blocks of one size, ranked by their maximal
// selection score; the `top` routes are taken from the `keep` leading blocks.
struct RouterSpec {
  int experts = 0, identity = 0, top = 0, count = 1, keep = 1;
};
constexpr int LM_MAX_ROUTES = 1024;  // experts + identity
constexpr int LM_MAX_TOP = 32;
// Routes rows of fp32 logits [rows][ld]: choice [rows][top] (router outputs, -1: none), weight [rows][top], rank
// [rows][top] = how many earlier arrivals the expert had, count [experts] += arrivals (csrc/moe.cu).
int moe_route(const float* logits, int64_t ld, const float* correction, int64_t rows, const RouterSpec& r, int* choice,
              float* weight, int* rank, int* count, cudaStream_t st);
// Copies the rows of h [rows][ld] of every chosen expert into blocks of 128 rows per expert: grouped [max rows][ld],
// slot [rows][top] (as in ResidualNorm), tile_group [max rows / 128] (the expert of a block or -1).
int moe_gather(const void* h, int dtype, int ld, int64_t rows, const RouterSpec& r, const int* choice, const int* rank,
               const int* count, void* grouped, int* slot, int* tile_group, int n_tiles, cudaStream_t st);
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
  float v[VPL];
  float m = -INFINITY;
#pragma unroll
  for (int j = 0; j < VPL; ++j) {
    const int i = j * 32 + lane;
    v[j] = i < n ? s[i] : -INFINITY;
    m = fmaxf(m, v[j]);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
  float sum = 0.f;
#pragma unroll
  for (int j = 0; j < VPL; ++j) {
    v[j] = j * 32 + lane < n ? expf(v[j] - m) : 0.f;
    sum += v[j];
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
  uint32_t key[VPL];
#pragma unroll
  for (int j = 0; j < VPL; ++j) {
    const int i = j * 32 + lane;
    key[j] = 0;
    if (i < n) {
      const float p = v[j] / sum, choice_score = p + correction[i];
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
struct DecodeInput {  // how a kernel obtains the vector it multiplies by, in every CTA
  // kind 0: h = norm(embedding of *id) * w_pre; 1: x = x_in + norm(y) * w_post, h = norm(x) * w_pre; 2: h = plain
  int kind = 2;
  const int* id = nullptr;
  const uint16_t* embed = nullptr;
  int vocab = 0;
  const float *x_in = nullptr, *y = nullptr, *w_post = nullptr, *w_pre = nullptr;
  float* x_out = nullptr;   // the new residual row (written by one CTA; another buffer than x_in)
  const float* plain = nullptr;
  int width = 0;            // channels the norms run over
  float eps = 0.f;
};
struct DecodeLinear {
  DecodeInput in;
  const uint16_t* w = nullptr;  // bf16 [n][k]
  int n = 0, k = 0;
  int epi = EPI_NONE;           // EPI_NONE or EPI_GELU_ERF
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
  const int* choice = nullptr;
  const float* weight = nullptr;
  const float* h = nullptr;     // [k]
  float* act = nullptr;         // [top][ff]
  float* out = nullptr;         // [k]
};
int decode_experts(const DecodeExperts& a, cudaStream_t st);

}  // namespace ytk
