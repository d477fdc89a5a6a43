// Mixture-of-experts routing for many tokens: one warp routes a token (warp_route, lm_ops.cuh), a second kernel copies
// the tokens of every expert into blocks of 128 rows for the grouped tensor-core products (linear_tc), and the
// residual kernel sums each token's experts in the order of choice (residual_norm). Which row of its expert's blocks a
// token gets depends on timing; its result does not.
#include "lm_ops.cuh"

namespace ytk {

constexpr int MR_WARPS = 4;

template <int VPL>
__global__ void __launch_bounds__(MR_WARPS * 32) moe_route_kernel(const float* logits, int64_t ld, const float* correction,
                                                                  int64_t rows, const RouterSpec r, int* choice,
                                                                  float* weight, int* rank, int* count) {
  extern __shared__ float route_s[];  // [MR_WARPS][2][experts + identity]
  dependent_wait();
  dependent_trigger();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n = r.experts + r.identity;
  float* s = route_s + warp * 2 * n;
  for (int64_t row = static_cast<int64_t>(blockIdx.x) * MR_WARPS + warp; row < rows;
       row += static_cast<int64_t>(gridDim.x) * MR_WARPS) {
    __syncwarp();
    for (int i = lane; i < n; i += 32) s[i] = logits[row * ld + i];
    __syncwarp();
    int c;
    float w;
    warp_route<VPL>(s, s + n, correction, r, lane, c, w);
    if (lane < r.top) {
      choice[row * r.top + lane] = c;
      weight[row * r.top + lane] = w;
      rank[row * r.top + lane] = (c >= 0 && c < r.experts) ? atomicAdd(count + c, 1) : 0;
    }
  }
}

int moe_route(const float* logits, int64_t ld, const float* correction, int64_t rows, const RouterSpec& r, int* choice,
              float* weight, int* rank, int* count, cudaStream_t st) {
  const int n = r.experts + r.identity;
  YTC_REQUIRE(r.experts >= 0 && r.identity >= 0 && n > 0 && n <= LM_MAX_ROUTES && r.top > 0 && r.top <= LM_MAX_TOP &&
                  r.top <= n && r.count > 0 && n % r.count == 0 && r.keep > 0 && r.keep <= r.count,
              "moe_route: %d + %d experts, top %d, %d of %d groups do not fit (at most %d routes, top %d)", r.experts,
              r.identity, r.top, r.keep, r.count, LM_MAX_ROUTES, LM_MAX_TOP);
  if (rows <= 0) return YTC_OK;
  const int64_t blocks = (rows + MR_WARPS - 1) / MR_WARPS, cap = static_cast<int64_t>(sm_count()) * 8;
  auto* fn = n <= 128 ? moe_route_kernel<4> : n <= 256 ? moe_route_kernel<8> : moe_route_kernel<LM_MAX_ROUTES / 32>;
  YTC_CUDA(launch_overlapped(fn, dim3(static_cast<unsigned>(blocks < cap ? blocks : cap)),
                             dim3(MR_WARPS * 32), MR_WARPS * 2 * n * sizeof(float), st, logits, ld, correction, rows, r,
                             choice, weight, rank, count));
  count_launch();
  YTC_CUDA(cudaGetLastError());
  return YTC_OK;
}

constexpr int MG_THREADS = 256;

// T: float or bf16 bits (of scaled copies; a plain copy moves 16-byte vectors whatever they hold).
template <typename T>
__global__ void __launch_bounds__(MG_THREADS) moe_gather_kernel(const MoeGather p) {
  extern __shared__ int first_tile[];  // [experts + 1]: first block of every expert
  __shared__ int warp_sum[MG_THREADS / 32];
  dependent_wait();
  dependent_trigger();
  const RouterSpec r = p.r;
  const int *count = p.count, n_tiles = p.n_tiles;
  int* tile_group = p.tile_group;
  // prefix sum of the blocks per expert, the same in every CTA
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int carry = 0;
  for (int e0 = 0; e0 < r.experts; e0 += MG_THREADS) {
    const int e = e0 + threadIdx.x;
    const int mine = e < r.experts ? (count[e] + LM_GROUP_ROWS - 1) / LM_GROUP_ROWS : 0;
    int inc = mine;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, inc, o);
      if (lane >= o) inc += v;
    }
    if (lane == 31) warp_sum[warp] = inc;
    __syncthreads();
    int before = carry, total = 0;
    for (int w = 0; w < MG_THREADS / 32; ++w) {
      if (w < warp) before += warp_sum[w];
      total += warp_sum[w];
    }
    if (e < r.experts) first_tile[e] = before + inc - mine;
    carry += total;
    __syncthreads();
  }
  if (threadIdx.x == 0) first_tile[r.experts] = carry;
  __syncthreads();
  if (blockIdx.x == 0) {
    for (int t = threadIdx.x; t < n_tiles; t += MG_THREADS) tile_group[t] = -1;
    __syncthreads();
    for (int e = threadIdx.x; e < r.experts; e += MG_THREADS)
      for (int t = first_tile[e]; t < first_tile[e + 1] && t < n_tiles; ++t) tile_group[t] = e;
  }
  const int64_t pairs = p.rows * r.top;
  const int row_vecs = p.ld * static_cast<int>(sizeof(T)) / 16;
  // one warp per (token, choice)
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * (MG_THREADS / 32) + warp; i < pairs;
       i += static_cast<int64_t>(gridDim.x) * (MG_THREADS / 32)) {
    const int c = p.choice[i];
    const int64_t row = i / r.top;
    if (c < 0 || c >= r.experts) {
      if (lane == 0) p.slot[i] = c < 0 ? -2 : -1;
      continue;
    }
    const int dst = first_tile[c] * LM_GROUP_ROWS + p.rank[i];
    if (lane == 0) p.slot[i] = dst;
    if (p.weight) {
      const float w = p.weight[i];
      const float* src = p.x + row * p.ld;
      T* out = static_cast<T*>(p.grouped) + static_cast<int64_t>(dst) * p.ld;
      for (int v = lane * 8; v < p.ld; v += 256) {
        float f[8];
        Vec8<float>::load(src + v, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] *= w;
        Vec8<T>::store(out + v, f);
      }
    } else {
      const uint4* src = static_cast<const uint4*>(p.h) + row * row_vecs;
      uint4* out = static_cast<uint4*>(p.grouped) + static_cast<int64_t>(dst) * row_vecs;
      for (int v = lane; v < row_vecs; v += 32) out[v] = src[v];
    }
  }
}

int moe_gather(const MoeGather& g, cudaStream_t st) {
  YTC_REQUIRE(g.ld % 8 == 0 && g.n_tiles >= moe_max_tiles(g.rows, g.r) && (!g.weight || g.x), "moe_gather: bad extent");
  if (g.rows <= 0) return YTC_OK;
  const int64_t blocks = (g.rows * g.r.top + MG_THREADS / 32 - 1) / (MG_THREADS / 32), cap = static_cast<int64_t>(sm_count()) * 8;
  YTC_CUDA(launch_overlapped(g.dtype == YTC_BF16 ? moe_gather_kernel<uint16_t> : moe_gather_kernel<float>,
                             dim3(static_cast<unsigned>(blocks < cap ? blocks : cap)), dim3(MG_THREADS),
                             (g.r.experts + 1) * sizeof(int), st, g));
  count_launch();
  YTC_CUDA(cudaGetLastError());
  return YTC_OK;
}

}  // namespace ytk
