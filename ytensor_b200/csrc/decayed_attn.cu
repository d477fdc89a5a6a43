// Linear attention with a decayed state (DecayedAttn, lm_ops.cuh), token by token.
#include "lm_ops.cuh"

namespace ytk {

// One CTA = (sequence, head, 16 value columns); the state's rows are spread over warps, lanes and RPT registers. Tokens come
// in blocks of DT_TOKENS; a block's outputs are summed over the warps once.
constexpr int DT_THREADS = 256, DT_WARPS = DT_THREADS / 32, DT_COLS = 16, DT_TOKENS = 16;

template <typename T, int RPT>
__global__ void __launch_bounds__(DT_THREADS) decayed_step_kernel(const DecayedAttn p) {
  extern __shared__ __align__(16) float dt_smem[];  // q, k [DT_TOKENS][dim] each
  __shared__ float v_s[DT_TOKENS][DT_COLS], part[DT_TOKENS][DT_WARPS][DT_COLS];
  float* q_s = dt_smem;
  float* k_s = dt_smem + DT_TOKENS * p.dim;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c0 = blockIdx.x * DT_COLS, h = blockIdx.y, b = blockIdx.z;
  const int cq = (lane & 3) * 4, rl = lane >> 2;  // four columns, row within 8
  const bool col_ok = c0 + cq < p.vdim;
  float* state = p.state + (static_cast<int64_t>(b) * p.heads + h) * p.dim * p.vdim + c0 + cq;
  const bool first = p.pos ? *p.pos == 0 : p.first;
  auto row_of = [&](int i) { return (i * DT_WARPS + warp) * 8 + rl; };
  float4 s[RPT];
#pragma unroll
  for (int i = 0; i < RPT; ++i) {  // (this call's state was written by an earlier call)
    const int r = row_of(i);
    s[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (!first && col_ok && r < p.dim) s[i] = *reinterpret_cast<const float4*>(state + static_cast<int64_t>(r) * p.vdim);
  }
  const float decay = p.decay[h];
  dependent_wait();
  dependent_trigger();
  const T *q = static_cast<const T*>(p.q), *k = static_cast<const T*>(p.k), *v = static_cast<const T*>(p.v);
  auto load = [](const T* at) { return sizeof(T) == 4 ? *reinterpret_cast<const float*>(at) : bf16_bits_to_f32(*reinterpret_cast<const uint16_t*>(at)); };
  for (int t0 = 0; t0 < p.len; t0 += DT_TOKENS) {
    const int n = p.len - t0 < DT_TOKENS ? p.len - t0 : DT_TOKENS;
    const int64_t row0 = static_cast<int64_t>(b) * p.len + t0;
    for (int i = threadIdx.x; i < n * p.dim; i += DT_THREADS) {
      const int t = i / p.dim, d = i - t * p.dim;
      const int64_t at = (row0 + t) * p.ld + static_cast<int64_t>(h) * p.dim + d;
      q_s[i] = load(q + at);
      k_s[i] = load(k + at);
    }
    for (int i = threadIdx.x; i < n * DT_COLS; i += DT_THREADS) {
      const int t = i / DT_COLS, c = i - t * DT_COLS;
      v_s[t][c] = c0 + c < p.vdim ? load(v + (row0 + t) * p.ld + static_cast<int64_t>(h) * p.vdim + c0 + c) : 0.f;
    }
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      const float4 vv = *reinterpret_cast<const float4*>(&v_s[t][cq]);
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int i = 0; i < RPT; ++i) {
        const int r = row_of(i);
        if (r >= p.dim) break;
        const float kk = k_s[t * p.dim + r], qq = q_s[t * p.dim + r];
        s[i].x = fmaf(decay, s[i].x, kk * vv.x); s[i].y = fmaf(decay, s[i].y, kk * vv.y);
        s[i].z = fmaf(decay, s[i].z, kk * vv.z); s[i].w = fmaf(decay, s[i].w, kk * vv.w);
        o.x = fmaf(qq, s[i].x, o.x); o.y = fmaf(qq, s[i].y, o.y);
        o.z = fmaf(qq, s[i].z, o.z); o.w = fmaf(qq, s[i].w, o.w);
      }
#pragma unroll
      for (int m = 4; m < 32; m <<= 1) {
        o.x += __shfl_xor_sync(0xffffffffu, o.x, m); o.y += __shfl_xor_sync(0xffffffffu, o.y, m);
        o.z += __shfl_xor_sync(0xffffffffu, o.z, m); o.w += __shfl_xor_sync(0xffffffffu, o.w, m);
      }
      if (lane < 4) *reinterpret_cast<float4*>(&part[t][warp][cq]) = o;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < n * DT_COLS; i += DT_THREADS) {
      const int t = i / DT_COLS, c = i - t * DT_COLS;
      if (c0 + c >= p.vdim) continue;
      float o = 0.f;
#pragma unroll
      for (int w = 0; w < DT_WARPS; ++w) o += part[t][w][c];
      const int64_t at = (row0 + t) * p.ld_o + static_cast<int64_t>(h) * p.vdim + c0 + c;
      if (sizeof(T) == 4) static_cast<float*>(p.o)[at] = o;
      else static_cast<uint16_t*>(p.o)[at] = bf16_rn_bits(o);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int r = row_of(i);
    if (col_ok && r < p.dim) *reinterpret_cast<float4*>(state + static_cast<int64_t>(r) * p.vdim) = s[i];
  }
}

template <typename T>
static int decayed_steps(const DecayedAttn& a, cudaStream_t st) {
  const int rpt = (a.dim + 8 * DT_WARPS - 1) / (8 * DT_WARPS);
  void (*fn)(DecayedAttn) = nullptr;
  if (rpt <= 1) fn = decayed_step_kernel<T, 1>;
  else if (rpt <= 2) fn = decayed_step_kernel<T, 2>;
  else if (rpt <= 4) fn = decayed_step_kernel<T, 4>;
  else if (rpt <= 8) fn = decayed_step_kernel<T, 8>;
  else {
    set_last_error("decayed_attention: heads of more than %d dimensions are not supported", 8 * 8 * DT_WARPS);
    return YTC_UNSUPPORTED;
  }
  const int smem = 2 * DT_TOKENS * a.dim * static_cast<int>(sizeof(float));
  const int s = ensure_dynamic_smem(reinterpret_cast<const void*>(fn), smem);
  if (s != YTC_OK) return s;
  YTC_CUDA(launch_overlapped(fn, dim3((a.vdim + DT_COLS - 1) / DT_COLS, a.heads, a.batch), dim3(DT_THREADS), smem, st, a));
  count_launch();
  YTC_CUDA(cudaGetLastError());
  return YTC_OK;
}

int decayed_attention(const DecayedAttn& a, cudaStream_t st) {
  if (a.len <= 0 || a.batch <= 0) return YTC_OK;
  YTC_REQUIRE(a.heads > 0 && a.dim > 0 && a.dim % 8 == 0 && a.vdim > 0 && a.vdim % 8 == 0 && (!a.pos || a.len == 1) &&
                  a.heads <= 65535 && a.batch <= 65535,
              "decayed_attention: bad extent");
  return a.dtype == YTC_BF16 ? decayed_steps<uint16_t>(a, st) : decayed_steps<float>(a, st);
}

}  // namespace ytk

using namespace ytk;

extern "C" int ytcuda_decayed_attn_fwd(int dtype, const void* q, const void* k, const void* v, int64_t ld, void* o,
                                       float* state, const float* decay, int batch, int len, int heads, int dim, int vdim,
                                       int first, int path, void* stream) {
  YTC_REQUIRE(dtype == YTC_F32 || dtype == YTC_BF16, "ytcuda_decayed_attn_fwd: dtype must be fp32 or bf16");
  YTC_REQUIRE(q && k && v && o && state && decay, "ytcuda_decayed_attn_fwd: null argument");
  YTC_REQUIRE(path >= 0 && path <= 2, "ytcuda_decayed_attn_fwd: path must be 0, 1 or 2");
  DecayedAttn a;
  a.dtype = dtype;
  a.q = q; a.k = k; a.v = v; a.ld = ld;
  a.o = o; a.ld_o = static_cast<int64_t>(heads) * vdim;
  a.state = state; a.decay = decay;
  a.batch = batch; a.len = len; a.heads = heads; a.dim = dim; a.vdim = vdim;
  a.first = first != 0;
  a.path = path;
  return decayed_attention(a, static_cast<cudaStream_t>(stream));
}
