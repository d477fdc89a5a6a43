// Row-wise kernels of the language models: embedding gather, residual stream with norms before and after a sublayer,
// K/V append with mixed values, and the fp32 linear layer with bf16 weights.
#include <math_constants.h>

#include "lm_ops.cuh"

namespace ytk {

// ------------------------------------------------------------------ embedding gather
// out[t, :] = scale * float(table[ids[t], :])   (scale 1: reference qwen3.cpp:378-385)
__global__ void __launch_bounds__(256) embedding_kernel(const uint16_t* table, const int* ids, float* out, int64_t n,
                                                        int hidden, int vocab, float scale) {
  const int per_row = hidden / 4;
  const int64_t total = n * per_row;
  for (int64_t i = blockIdx.x * static_cast<int64_t>(blockDim.x) + threadIdx.x; i < total;
       i += static_cast<int64_t>(gridDim.x) * blockDim.x) {
    const int64_t t = i / per_row;
    const int c = static_cast<int>(i - t * per_row) * 4;
    int id = ids[t];
    id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
    const uint2 w = *reinterpret_cast<const uint2*>(table + static_cast<int64_t>(id) * hidden + c);
    float4 o;
    o.x = scale * bf16_bits_to_f32(static_cast<uint16_t>(w.x & 0xFFFF));
    o.y = scale * bf16_bits_to_f32(static_cast<uint16_t>(w.x >> 16));
    o.z = scale * bf16_bits_to_f32(static_cast<uint16_t>(w.y & 0xFFFF));
    o.w = scale * bf16_bits_to_f32(static_cast<uint16_t>(w.y >> 16));
    *reinterpret_cast<float4*>(out + t * hidden + c) = o;
  }
}

int embed_rows(const uint16_t* table, const int* ids, float* x, int64_t rows, int width, int vocab, float scale,
               cudaStream_t st) {
  if (rows <= 0) return YTC_OK;
  const int64_t blocks = (rows * (width / 4) + 255) / 256, cap = static_cast<int64_t>(sm_count()) * 16;
  embedding_kernel<<<static_cast<unsigned>(blocks < cap ? blocks : cap), 256, 0, st>>>(table, ids, x, rows, width, vocab, scale);
  count_launch();
  YTC_CUDA(cudaGetLastError());
  return YTC_OK;
}

// ------------------------------------------------------------------ residual stream
constexpr int RN_THREADS = 256;

__device__ __forceinline__ float rn_block_sum(float v, float* red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < RN_THREADS / 32; ++i) t += red[i];
  return t;
}

// VPT: float4 slots per thread (the row stays in registers between the two norms).
template <typename T, int VPT>
__global__ void __launch_bounds__(RN_THREADS) residual_norm_kernel(const ResidualNorm p) {
  __shared__ float red[2][RN_THREADS / 32];
  __shared__ int s_slot[LM_MAX_TOP];
  __shared__ float s_weight[LM_MAX_TOP];
  dependent_wait();
  dependent_trigger();
  const int64_t row = p.row_index ? p.row_index[blockIdx.x] : blockIdx.x;
  float* x = p.x + row * p.ld;
  const int nv = p.ld / 4;
  float4 xv[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * RN_THREADS;
    xv[i] = c < nv ? reinterpret_cast<const float4*>(x)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  if (p.w_post) {
    float4 yv[VPT];
    if (p.slot) {
      if (threadIdx.x < p.top) {
        s_slot[threadIdx.x] = p.slot[row * p.top + threadIdx.x];
        s_weight[threadIdx.x] = p.weight ? p.weight[row * p.top + threadIdx.x] : 1.f;
      }
      __syncthreads();
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + i * RN_THREADS;
        yv[i] = p.y && c < nv ? reinterpret_cast<const float4*>(p.y + row * p.ld)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
      }
      for (int k = 0; k < p.top; ++k) {  // in the order of choice: the sum does not depend on the batch
        const int s = s_slot[k];
        if (s < -1) continue;
        const T* src = s >= 0 ? static_cast<const T*>(p.expert_out) + static_cast<int64_t>(s) * p.ld
                              : static_cast<const T*>(p.h_in) + row * p.ld;
        const float w = s_weight[k];
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
          const int c = threadIdx.x + i * RN_THREADS;
          if (c >= nv) continue;
          float4 e;
          if (sizeof(T) == 4) {
            e = reinterpret_cast<const float4*>(src)[c];
          } else {
            const uint2 u = reinterpret_cast<const uint2*>(src)[c];
            e = make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xFFFF0000u), __uint_as_float(u.y << 16),
                            __uint_as_float(u.y & 0xFFFF0000u));
          }
          yv[i].x = fmaf(w, e.x, yv[i].x); yv[i].y = fmaf(w, e.y, yv[i].y);
          yv[i].z = fmaf(w, e.z, yv[i].z); yv[i].w = fmaf(w, e.w, yv[i].w);
        }
      }
    } else {
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + i * RN_THREADS;
        yv[i] = c < nv ? reinterpret_cast<const float4*>(p.y + row * p.ld)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
      }
    }
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      ss = fmaf(yv[i].x, yv[i].x, ss); ss = fmaf(yv[i].y, yv[i].y, ss);
      ss = fmaf(yv[i].z, yv[i].z, ss); ss = fmaf(yv[i].w, yv[i].w, ss);
    }
    const float inv = 1.0f / sqrtf(rn_block_sum(ss, red[0]) / p.width + p.eps);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * RN_THREADS;
      if (c >= nv) continue;
      const float4 g = reinterpret_cast<const float4*>(p.w_post)[c];
      xv[i].x += yv[i].x * inv * g.x; xv[i].y += yv[i].y * inv * g.y;
      xv[i].z += yv[i].z * inv * g.z; xv[i].w += yv[i].w * inv * g.w;
      reinterpret_cast<float4*>(x)[c] = xv[i];
    }
  }
  if (!p.h) return;
  T* h = static_cast<T*>(p.h) + static_cast<int64_t>(blockIdx.x) * p.ld;
  if (!p.w_pre) {
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * RN_THREADS;
      if (c >= nv) continue;
      if (sizeof(T) == 4) reinterpret_cast<float4*>(h)[c] = xv[i];
      else reinterpret_cast<uint2*>(h)[c] = make_uint2(pack_bf16x2_rn(xv[i].x, xv[i].y), pack_bf16x2_rn(xv[i].z, xv[i].w));
    }
    return;
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    ss = fmaf(xv[i].x, xv[i].x, ss); ss = fmaf(xv[i].y, xv[i].y, ss);
    ss = fmaf(xv[i].z, xv[i].z, ss); ss = fmaf(xv[i].w, xv[i].w, ss);
  }
  const float inv = 1.0f / sqrtf(rn_block_sum(ss, red[1]) / p.width + p.eps);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * RN_THREADS;
    if (c >= nv) continue;
    const float4 g = reinterpret_cast<const float4*>(p.w_pre)[c];
    const float4 o = make_float4(xv[i].x * inv * g.x, xv[i].y * inv * g.y, xv[i].z * inv * g.z, xv[i].w * inv * g.w);
    if (sizeof(T) == 4) reinterpret_cast<float4*>(h)[c] = o;
    else reinterpret_cast<uint2*>(h)[c] = make_uint2(pack_bf16x2_rn(o.x, o.y), pack_bf16x2_rn(o.z, o.w));
  }
}

template <typename T>
static int residual_norm_t(const ResidualNorm& a, cudaStream_t st) {
  const int vpt = (a.ld / 4 + RN_THREADS - 1) / RN_THREADS;
  void (*fn)(ResidualNorm) = nullptr;
  if (vpt <= 1) fn = residual_norm_kernel<T, 1>;
  else if (vpt <= 2) fn = residual_norm_kernel<T, 2>;
  else if (vpt <= 4) fn = residual_norm_kernel<T, 4>;
  else if (vpt <= 8) fn = residual_norm_kernel<T, 8>;
  else {
    set_last_error("residual_norm: rows of more than %d channels are not supported", 8 * 4 * RN_THREADS);
    return YTC_UNSUPPORTED;
  }
  YTC_CUDA(launch_overlapped(fn, dim3(static_cast<unsigned>(a.rows)), dim3(RN_THREADS), 0, st, a));
  count_launch();
  YTC_CUDA(cudaGetLastError());
  return YTC_OK;
}

int residual_norm(const ResidualNorm& a, cudaStream_t st) {
  if (a.rows <= 0) return YTC_OK;
  YTC_REQUIRE(a.ld % 8 == 0 && a.width > 0 && a.width <= a.ld && a.top <= LM_MAX_TOP, "residual_norm: bad extent");
  return a.dtype == YTC_BF16 ? residual_norm_t<uint16_t>(a, st) : residual_norm_t<float>(a, st);
}

// ------------------------------------------------------------------ output gate
// One row per CTA, pieces of 8 elements per thread; without a norm a row's pieces are independent.
template <typename T, int VPT>
__global__ void __launch_bounds__(RN_THREADS) gated_rows_kernel(const GatedRows p) {
  __shared__ float red[RN_THREADS / 32];
  dependent_wait();
  dependent_trigger();
  const int64_t row = blockIdx.x;
  const T* in = static_cast<const T*>(p.in) + row * p.ld_in;
  const T* gate = static_cast<const T*>(p.gate) + row * p.ld_gate;
  T* out = static_cast<T*>(p.out) + row * p.ld_out;
  const int nv = p.cols / 8;
  float f[VPT][8];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * RN_THREADS;
    if (c >= nv) continue;
    Vec8<T>::load(in + c * 8, f[i]);
#pragma unroll
    for (int e = 0; e < 8; ++e) ss = fmaf(f[i][e], f[i][e], ss);
  }
  float inv = 1.f;
  if (p.w) inv = 1.0f / sqrtf(rn_block_sum(ss, red) / p.width + p.eps);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * RN_THREADS;
    if (c >= nv) continue;
    float g[8];
    if (p.w) {
      Vec8<float>::load(p.w + c * 8, g);
#pragma unroll
      for (int e = 0; e < 8; ++e) f[i][e] *= inv * g[e];
    }
    Vec8<T>::load(gate + c * 8, g);
#pragma unroll
    for (int e = 0; e < 8; ++e) f[i][e] *= sizeof(T) == 4 ? lm_sigmoid(g[e]) : lm_sigmoid_fast(g[e]);
    Vec8<T>::store(out + c * 8, f[i]);
  }
}

template <typename T>
static int gated_rows_t(const GatedRows& a, cudaStream_t st) {
  const int vpt = (a.cols / 8 + RN_THREADS - 1) / RN_THREADS;
  void (*fn)(GatedRows) = nullptr;
  if (vpt <= 1) fn = gated_rows_kernel<T, 1>;
  else if (vpt <= 2) fn = gated_rows_kernel<T, 2>;
  else if (vpt <= 4) fn = gated_rows_kernel<T, 4>;
  else if (vpt <= 8) fn = gated_rows_kernel<T, 8>;
  else {
    set_last_error("gated_rows: rows of more than %d channels are not supported", 8 * 8 * RN_THREADS);
    return YTC_UNSUPPORTED;
  }
  YTC_CUDA(launch_overlapped(fn, dim3(static_cast<unsigned>(a.rows)), dim3(RN_THREADS), 0, st, a));
  count_launch();
  YTC_CUDA(cudaGetLastError());
  return YTC_OK;
}

int gated_rows(const GatedRows& a, cudaStream_t st) {
  if (a.rows <= 0) return YTC_OK;
  YTC_REQUIRE(a.cols > 0 && a.cols % 8 == 0 && a.ld_in % 8 == 0 && a.ld_gate % 8 == 0 && a.ld_out % 8 == 0 &&
                  (!a.w || (a.width > 0 && a.width <= a.cols)),
              "gated_rows: bad extent");
  return a.dtype == YTC_BF16 ? gated_rows_t<uint16_t>(a, st) : gated_rows_t<float>(a, st);
}

// ------------------------------------------------------------------ K/V append
// One row (token) per CTA at a time, one 8-element piece of a key or value vector per thread.
constexpr int AK_THREADS = 128;
template <typename T>
__global__ void __launch_bounds__(AK_THREADS) append_kv_kernel(const AppendKv p) {
  dependent_wait();
  dependent_trigger();
  const int kp = p.kv_heads * p.dim / 8, vp = p.kv_heads * p.vdim / 8;
  const int rows = p.batch * p.len;
  const float lam = p.mix == VMIX_MIX ? *p.lambda : 0.f;
  for (int row = blockIdx.x; row < rows; row += gridDim.x) {
    const int b = row / p.len, t = row - b * p.len;
    const int64_t ring_row = (p.pos0 + t) % p.ring;
    const T* src = static_cast<const T*>(p.qkv) + row * p.ld;
    for (int c = threadIdx.x; c < kp + vp; c += AK_THREADS) {
      float f[8];
      if (c < kp) {
        const int e = c * 8, g = e / p.dim, d = e - g * p.dim;
        Vec8<T>::load(src + p.k_off + e, f);
        Vec8<T>::store(static_cast<T*>(p.k) + ((static_cast<int64_t>(b) * p.kv_heads + g) * p.ring + ring_row) * p.dim + d, f);
      } else {
        const int e = (c - kp) * 8, g = e / p.vdim, d = e - g * p.vdim;
        Vec8<T>::load(src + p.v_off + e, f);
        T* first = static_cast<T*>(p.v_first) + row * (static_cast<int64_t>(p.kv_heads) * p.vdim) + e;
        if (p.mix == VMIX_FIRST) Vec8<T>::store(first, f);
        if (p.mix == VMIX_MIX) {
          float v0[8];
          Vec8<T>::load(first, v0);
#pragma unroll
          for (int k = 0; k < 8; ++k) f[k] = (1.f - lam) * f[k] + lam * v0[k];
        }
        Vec8<T>::store(static_cast<T*>(p.v) + ((static_cast<int64_t>(b) * p.kv_heads + g) * p.ring + ring_row) * p.vdim + d, f);
      }
    }
  }
}

int append_kv(const AppendKv& a, cudaStream_t st) {
  YTC_REQUIRE(a.dim % 8 == 0 && a.vdim % 8 == 0 && a.ld % 8 == 0 && a.k_off % 8 == 0 && a.v_off % 8 == 0 && a.len <= a.ring,
              "append_kv: bad extent");
  YTC_REQUIRE(a.mix == VMIX_NONE || a.v_first, "append_kv: no place for the first layer's values");
  const int64_t blocks = static_cast<int64_t>(a.batch) * a.len, cap = static_cast<int64_t>(sm_count()) * 16;
  YTC_CUDA(launch_overlapped(a.dtype == YTC_BF16 ? append_kv_kernel<uint16_t> : append_kv_kernel<float>,
                             dim3(static_cast<unsigned>(blocks < cap ? blocks : cap)), dim3(AK_THREADS), 0, st, a));
  count_launch();
  YTC_CUDA(cudaGetLastError());
  return YTC_OK;
}

// ------------------------------------------------------------------ fp32 linear, bf16 weights, FFMA
// 64 x 64 outputs per CTA, 4 x 4 per thread, k in steps of 16. The sum over k runs in one fixed order for every row.
constexpr int LF_BM = 64, LF_BN = 64, LF_BK = 16;
struct LinearF32Params {
  const float* x;
  const uint16_t* w;
  float* y;
  int64_t ldx, ldw, ldy;
  int m, n, k;
  LinearEpilogue ex;
};
__global__ void __launch_bounds__(256) linear_f32_kernel(const LinearF32Params p) {
  __shared__ float xs[LF_BK][LF_BM + 4], ws[LF_BK][LF_BN + 4];
  dependent_wait();
  dependent_trigger();
  const int m0 = blockIdx.y * LF_BM, n0 = blockIdx.x * LF_BN;
  int64_t w_row0 = 0;
  if (p.ex.tile_group) {
    const int g = p.ex.tile_group[m0 / LM_GROUP_ROWS];
    if (g < 0) return;
    w_row0 = static_cast<int64_t>(g) * p.n;
  }
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lr = threadIdx.x >> 2, lc = (threadIdx.x & 3) * 4;  // loader: row of the tile, first of 4 columns
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.k; k0 += LF_BK) {
    float4 xv = make_float4(0.f, 0.f, 0.f, 0.f);
    uint2 wv = make_uint2(0u, 0u);
    if (m0 + lr < p.m && k0 + lc < p.k) xv = *reinterpret_cast<const float4*>(p.x + (m0 + lr) * p.ldx + k0 + lc);
    if (n0 + lr < p.n && k0 + lc < p.k)
      wv = *reinterpret_cast<const uint2*>(p.w + (w_row0 + n0 + lr) * p.ldw + k0 + lc);
    __syncthreads();
    xs[lc][lr] = xv.x; xs[lc + 1][lr] = xv.y; xs[lc + 2][lr] = xv.z; xs[lc + 3][lr] = xv.w;
    ws[lc][lr] = __uint_as_float(wv.x << 16); ws[lc + 1][lr] = __uint_as_float(wv.x & 0xFFFF0000u);
    ws[lc + 2][lr] = __uint_as_float(wv.y << 16); ws[lc + 3][lr] = __uint_as_float(wv.y & 0xFFFF0000u);
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < LF_BK; ++kk) {
      const float4 a = *reinterpret_cast<const float4*>(&xs[kk][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&ws[kk][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= p.m) continue;
    if (p.ex.epi == EPI_SWIGLU_PAIRS || p.ex.epi == EPI_CLAMP_PAIRS) {
#pragma unroll
      for (int j = 0; j < 4; j += 2) {
        const int n = n0 + tx * 4 + j;
        if (n + 1 < p.n) p.y[m * p.ldy + n / 2] = lm_gated(p.ex, acc[i][j], acc[i][j + 1]);
      }
      continue;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n < p.n) p.y[m * p.ldy + n] = lm_activation(p.ex, acc[i][j], n);
    }
  }
}

int linear_f32(const float* x, int64_t ldx, const uint16_t* w, int64_t ldw, float* y, int64_t ldy, int m, int n, int k,
               const LinearEpilogue& ex, cudaStream_t st) {
  if (m <= 0 || n <= 0) return YTC_OK;
  YTC_REQUIRE(k % 4 == 0 && ldx % 4 == 0 && ldw % 4 == 0, "linear_f32: rows must be whole groups of four elements");
  YTC_REQUIRE(!epi_pairs(ex.epi) || n % 2 == 0, "linear_f32: an odd number of gate / up rows");
  const int64_t tm = (static_cast<int64_t>(m) + LF_BM - 1) / LF_BM;
  YTC_REQUIRE(tm <= 65535, "linear_f32: too many rows");
  LinearF32Params p{x, w, y, ldx, ldw, ldy, m, n, k, ex};
  YTC_CUDA(launch_overlapped(linear_f32_kernel, dim3((n + LF_BN - 1) / LF_BN, static_cast<unsigned>(tm)), dim3(256), 0, st, p));
  count_launch();
  YTC_CUDA(cudaGetLastError());
  return YTC_OK;
}

}  // namespace ytk

using namespace ytk;

extern "C" {

int ytcuda_embedding(const void* table_bf16, const int32_t* ids, float* out, int64_t n, int hidden, int vocab,
                     void* stream) {
  YTC_REQUIRE(n >= 0 && hidden >= 0 && vocab > 0, "ytcuda_embedding: bad extent");
  if (n == 0 || hidden == 0) return YTC_OK;
  YTC_REQUIRE(table_bf16 && ids && out, "ytcuda_embedding: null tensor");
  YTC_REQUIRE(hidden % 4 == 0, "ytcuda_embedding: hidden must be a multiple of 4");
  return embed_rows(static_cast<const uint16_t*>(table_bf16), ids, out, n, hidden, vocab, 1.f,
                    static_cast<cudaStream_t>(stream));
}

}  // extern "C"
