// Linear attention with a decayed state (DecayedAttn, lm_ops.cuh).
//
// Token by token (decayed_step_kernel): fp32 products, any sizes, decode steps and short inputs.
// In chunks of 128 tokens (bf16, heads of 128 x 128) on tcgen05. With w = decay and the state S before a chunk of n tokens,
//   o_t = w^(t+1) S^T q_t + sum over s <= t of w^(t-s) (q_t . k_s) v_s,   S' = w^n S + sum over s < n of w^(n-1-s) k_s v_s^T:
// one launch forms every chunk's own contribution to the state (all chunks at once), an elementwise scan over the chunks
// turns these into the states before each chunk, a third launch computes all chunks' outputs. Whatever carries a decay
// (state, weights, decayed values) enters a product as two bf16 numbers, hi + lo, with 16 mantissa bits together.
#include <algorithm>

#include "lm_ops.cuh"
#include "ptx_sm100.cuh"

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

// ------------------------------------------------------------------ chunks of 128 tokens, heads of 128 x 128
constexpr int DC = 128;                      // tokens of a chunk = head dims
constexpr int DC_BOX = DC * 128;             // bytes of 128 rows x 64 bf16 columns, 128-byte swizzle
constexpr int DC_TILE = 2 * DC_BOX;
constexpr int DC_STATE = DC * DC;            // elements of a state

struct DecayedChunks {
  const float* own;     // [units][DC][DC] fp32: a chunk's own contribution to the state
  uint16_t* planes;     // [units][2][DC][DC] bf16: the state before the chunk, hi and lo
  const float* decay;
  float* state;         // [batch][heads][DC][DC]
  int heads, chunks, len, first;
  int* status;
  // unit of (batch, head, chunk)
  __device__ __forceinline__ int64_t unit(int b, int h, int c) const {
    return (static_cast<int64_t>(b) * heads + h) * chunks + c;
  }
};

// w^i for i <= DC, in shared memory
__device__ __forceinline__ void decay_powers(float* pw, float w) {
  const float l2 = log2f(fabsf(w));
  for (int i = threadIdx.x; i <= DC; i += blockDim.x) {
    const float v = exp2f(static_cast<float>(i) * l2);
    pw[i] = i == 0 ? 1.f : (w < 0.f && (i & 1)) ? -v : v;
  }
}
__device__ __forceinline__ void load_tile(uint8_t* dst, const CUtensorMap* m, uint64_t* bar, int row, int head, int batch) {
  tma_load_4d(dst, m, bar, 0, row, head, batch);
  tma_load_4d(dst + DC_BOX, m, bar, 64, row, head, batch);
}
// hi + lo of a pair of floats, packed
__device__ __forceinline__ void split_pair(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2_rn(a, b);
  lo = pack_bf16x2_rn(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xFFFF0000u));
}
// A wait that gave up leaves copies in flight: they get a bounded drain before the CTA ends.
__device__ __forceinline__ void drain(uint64_t* bar) {
  const long long t0 = clock64();
  while (!mbar_try_wait(bar, 0) && clock64() - t0 < 20000000ll) {
  }
}

// own = sum over s of k_s (w^(n-1-s) v_s)^T: K^T is the M operand (dims x tokens, unit stride along the dims), the decayed
// values the N operand.
constexpr int DS_THREADS = 256;
constexpr int DS_SMEM = 3 * DC_TILE + 1024;
__global__ void __launch_bounds__(DS_THREADS, 2) decayed_chunk_state_kernel(const __grid_constant__ CUtensorMap tmK,
                                                                            const __grid_constant__ CUtensorMap tmV,
                                                                            const __grid_constant__ CUtensorMap tmU,
                                                                            const DecayedChunks p) {
  extern __shared__ uint8_t ds_raw[];
  __shared__ uint64_t bars[2];
  __shared__ uint32_t tmem_slot;
  __shared__ int abort_flag;
  __shared__ float pw[DC + 1];
  uint8_t* smem = ds_raw + ((1024u - (smem_u32(ds_raw) & 1023u)) & 1023u);
  uint8_t *k_s = smem, *v_hi = smem + DC_TILE, *v_lo = smem + 2 * DC_TILE;
  volatile int* abort_word = &abort_flag;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  const int n = p.len - c * DC < DC ? p.len - c * DC : DC;
  if (threadIdx.x == 0) {
    mbar_init(&bars[0], 1);
    mbar_init(&bars[1], 1);
    abort_flag = 0;
    fence_mbar_init();
    fence_proxy_async_smem();
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
  }
  if (warp == 1) {
    tmem_alloc(&tmem_slot, 128);
    tmem_relinquish();
  }
  decay_powers(pw, p.decay[h]);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t t_d = tmem_slot;
  dependent_wait();
  dependent_trigger();
  if (threadIdx.x == 0) {  // (tokens behind the input's end arrive as zeros)
    mbar_expect_tx(&bars[0], 2 * DC_TILE);
    load_tile(v_hi, &tmV, &bars[0], c * DC, h, b);
    load_tile(k_s, &tmK, &bars[0], c * DC, h, b);
  }
  bool ok = mbar_wait(&bars[0], 0, abort_word);
  if (__syncthreads_and(ok)) {
    // (a row of a box is one token's 128 bytes wherever the swizzle puts its pieces)
    for (int i = threadIdx.x; i < DC_TILE / 16; i += DS_THREADS) {
      const int t = (i & (DC_BOX / 16 - 1)) >> 3;
      const float f = t < n ? pw[n - 1 - t] : 0.f;
      float v[8];
      Vec8<uint16_t>::load(reinterpret_cast<const uint16_t*>(v_hi + i * 16), v);
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) split_pair(f * v[2 * e], f * v[2 * e + 1], hi[e], lo[e]);
      *reinterpret_cast<uint4*>(v_hi + i * 16) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      *reinterpret_cast<uint4*>(v_lo + i * 16) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
    fence_proxy_async_smem();
    __syncthreads();
    if (threadIdx.x == 0) {
      const uint32_t idesc = umma_idesc(1u, 1, 1, DC, DC);
      const uint32_t ka = smem_u32(k_s), va = smem_u32(v_hi), vb = smem_u32(v_lo);
#pragma unroll
      for (int kk = 0; kk < DC / 16; ++kk)
        tc_mma_f16(t_d, umma_smem_desc_sw128(ka + kk * 2048, DC_BOX, 1024), umma_smem_desc_sw128(va + kk * 2048, DC_BOX, 1024),
                   idesc, kk != 0 ? 1u : 0u);
#pragma unroll
      for (int kk = 0; kk < DC / 16; ++kk)
        tc_mma_f16(t_d, umma_smem_desc_sw128(ka + kk * 2048, DC_BOX, 1024), umma_smem_desc_sw128(vb + kk * 2048, DC_BOX, 1024),
                   idesc, 1u);
      tc_commit(&bars[1]);
    }
    ok = mbar_wait(&bars[1], 0, abort_word);
    tc_fence_after();
    if (__syncthreads_and(ok)) {
      // rows of 32 floats in the store's 128-byte swizzle, over the operands that have been read
      const int t = (warp & 3) * 32 + lane;
#pragma unroll
      for (int q = (warp >> 2) * 2; q < (warp >> 2) * 2 + 2; ++q) {
        uint32_t r[32];
        tmem_ld_32x32b_x32(t_d + q * 32 + (static_cast<uint32_t>((warp & 3) * 32) << 16), r);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 8; ++j)
          *reinterpret_cast<uint4*>(smem + q * DC_BOX + t * 128 + ((j ^ (t & 7)) << 4)) =
              make_uint4(r[4 * j], r[4 * j + 1], r[4 * j + 2], r[4 * j + 3]);
      }
      fence_proxy_async_smem();
      __syncthreads();
      if (threadIdx.x == 0) {
        const int row = static_cast<int>(p.unit(b, h, c) * DC);
#pragma unroll
        for (int q = 0; q < 4; ++q) tma_store_2d(&tmU, smem + q * DC_BOX, q * 32, row);
        tma_store_commit();
        tma_store_wait_all<0>();
      }
    }
  } else if (threadIdx.x == 0) {
    drain(&bars[0]);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(t_d, 128);
  }
  if (threadIdx.x == 0 && abort_flag) atomicExch(p.status, YTC_TIMEOUT);
}

// States before every chunk, and the state behind the last one. Four elements per thread.
constexpr int DN_THREADS = 256;
__global__ void __launch_bounds__(DN_THREADS) decayed_chunk_scan_kernel(const DecayedChunks p) {
  const int h = blockIdx.y, b = blockIdx.z;
  const int at = (blockIdx.x * DN_THREADS + threadIdx.x) * 4;
  float* state = p.state + (static_cast<int64_t>(b) * p.heads + h) * DC_STATE + at;
  float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
  if (!p.first) s = *reinterpret_cast<const float4*>(state);
  const float w = p.decay[h];
  const int n_last = p.len - (p.chunks - 1) * DC;
  auto power = [&](int n) {
    const float v = exp2f(static_cast<float>(n) * log2f(fabsf(w)));
    return (w < 0.f && (n & 1)) ? -v : v;
  };
  const float full = power(DC), last = power(n_last);
  dependent_wait();
  dependent_trigger();
  const float* own = p.own + p.unit(b, h, 0) * DC_STATE + at;
  uint16_t* planes = p.planes + p.unit(b, h, 0) * 2 * DC_STATE + at;
#pragma unroll 4
  for (int c = 0; c < p.chunks; ++c) {
    const float4 u = *reinterpret_cast<const float4*>(own + static_cast<int64_t>(c) * DC_STATE);
    uint2 hi, lo;
    split_pair(s.x, s.y, hi.x, lo.x);
    split_pair(s.z, s.w, hi.y, lo.y);
    uint16_t* out = planes + static_cast<int64_t>(c) * 2 * DC_STATE;
    *reinterpret_cast<uint2*>(out) = hi;
    *reinterpret_cast<uint2*>(out + DC_STATE) = lo;
    const float f = c + 1 < p.chunks ? full : last;
    s.x = fmaf(f, s.x, u.x); s.y = fmaf(f, s.y, u.y); s.z = fmaf(f, s.z, u.z); s.w = fmaf(f, s.w, u.w);
  }
  *reinterpret_cast<float4*>(state) = s;
}

// Outputs of one chunk. One warp loads and issues: S = Q K^T, then, over K's place in shared memory, the state before the
// chunk (hi, lo) for C = Q S; eight warps turn S into the decayed lower triangle P (hi, lo) in tensor memory, over S, and
// take C into registers; P V goes over C. Three tiles of shared memory and half of tensor memory: two CTAs per SM.
constexpr int DO_WORKERS = 256, DO_THREADS = DO_WORKERS + 32;
constexpr int DO_SMEM = 3 * DC_TILE + 1024;
enum { DO_QK = 0, DO_V, DO_STATE, DO_S, DO_HI_DONE, DO_C, DO_P, DO_O, DO_BARS };
__device__ __forceinline__ void workers_sync() { asm volatile("bar.sync 1, %0;" ::"n"(DO_WORKERS) : "memory"); }
__global__ void __launch_bounds__(DO_THREADS, 2) decayed_chunk_out_kernel(const __grid_constant__ CUtensorMap tmQ,
                                                                          const __grid_constant__ CUtensorMap tmK,
                                                                          const __grid_constant__ CUtensorMap tmV,
                                                                          const __grid_constant__ CUtensorMap tmS,
                                                                          const __grid_constant__ CUtensorMap tmO,
                                                                          const DecayedChunks p) {
  extern __shared__ uint8_t do_raw[];
  __shared__ uint64_t bars[DO_BARS];
  __shared__ uint32_t tmem_slot;
  __shared__ int abort_flag;
  __shared__ float pw[DC + 1];
  uint8_t* smem = do_raw + ((1024u - (smem_u32(do_raw) & 1023u)) & 1023u);
  uint8_t *q_s = smem, *k_s = smem + DC_TILE, *v_s = smem + 2 * DC_TILE;
  volatile int* abort_word = &abort_flag;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  const bool carried = c > 0 || !p.first;  // (the state before the first chunk of a sequence is zero)
  if (threadIdx.x == 0) {
    for (int i = 0; i < DO_BARS; ++i) mbar_init(&bars[i], i == DO_P ? DO_WORKERS / 32 : 1);
    abort_flag = 0;
    fence_mbar_init();
    fence_proxy_async_smem();
  }
  if (warp == DO_WORKERS / 32) {
    tmem_alloc(&tmem_slot, 256);
    tmem_relinquish();
  }
  decay_powers(pw, p.decay[h]);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t t_s = tmem_slot, t_o = t_s + 128, t_hi = t_s, t_lo = t_s + 64;
  dependent_wait();
  dependent_trigger();
  if (warp == DO_WORKERS / 32) {
    if (lane == 0) {
      mbar_expect_tx(&bars[DO_QK], 2 * DC_TILE);
      load_tile(q_s, &tmQ, &bars[DO_QK], c * DC, h, b);
      load_tile(k_s, &tmK, &bars[DO_QK], c * DC, h, b);
      mbar_expect_tx(&bars[DO_V], DC_TILE);
      load_tile(v_s, &tmV, &bars[DO_V], c * DC, h, b);
      const uint32_t qa = smem_u32(q_s), ka = smem_u32(k_s), va = smem_u32(v_s);
      bool ok = mbar_wait(&bars[DO_QK], 0, abort_word);
      if (ok) {
        const uint32_t idesc = umma_idesc(1u, 0, 0, DC, DC);
#pragma unroll
        for (int kk = 0; kk < DC / 16; ++kk) {
          const uint32_t off = (kk >> 2) * DC_BOX + (kk & 3) * 32;
          tc_mma_f16(t_s, umma_smem_desc_sw128(qa + off, 16, 1024), umma_smem_desc_sw128(ka + off, 16, 1024), idesc,
                     kk != 0 ? 1u : 0u);
        }
        tc_commit(&bars[DO_S]);
      }
      if (carried) {
        const uint32_t idesc = umma_idesc(1u, 0, 1, DC, DC);
        const int row = static_cast<int>(p.unit(b, h, c) * 2 * DC);
#pragma unroll 1
        for (int i = 0; i < 2 && ok; ++i) {  // (what stood in K's place has been read: S, then C's first half, are done)
          ok = mbar_wait(&bars[i == 0 ? DO_S : DO_HI_DONE], 0, abort_word);
          if (!ok) break;
          mbar_expect_tx(&bars[DO_STATE], DC_TILE);
          tma_load_2d(k_s, &tmS, &bars[DO_STATE], 0, row + i * DC);
          tma_load_2d(k_s + DC_BOX, &tmS, &bars[DO_STATE], 64, row + i * DC);
          ok = mbar_wait(&bars[DO_STATE], static_cast<uint32_t>(i), abort_word);
          if (!ok) break;
#pragma unroll
          for (int kk = 0; kk < DC / 16; ++kk) {
            const uint32_t off = (kk >> 2) * DC_BOX + (kk & 3) * 32;
            tc_mma_f16(t_o, umma_smem_desc_sw128(qa + off, 16, 1024), umma_smem_desc_sw128(ka + kk * 2048, DC_BOX, 1024), idesc,
                       (i != 0 || kk != 0) ? 1u : 0u);
          }
          tc_commit(&bars[i == 0 ? DO_HI_DONE : DO_C]);
        }
      }
      ok = ok && mbar_wait(&bars[DO_V], 0, abort_word) && mbar_wait(&bars[DO_P], 0, abort_word);
      if (ok) {
        tc_fence_after();
        const uint32_t idesc = umma_idesc(1u, 0, 1, DC, DC);
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
          for (int kk = 0; kk < DC / 16; ++kk)
            tc_mma_f16_ts(t_o, (i ? t_lo : t_hi) + kk * 8, umma_smem_desc_sw128(va + kk * 2048, DC_BOX, 1024), idesc,
                          (i != 0 || kk != 0) ? 1u : 0u);
        tc_commit(&bars[DO_O]);
      } else {
        drain(&bars[DO_QK]);
        drain(&bars[DO_V]);
      }
    }
    __syncwarp();
  } else {
    // warps 0 - 3 take the first 64 columns of their rows, warps 4 - 7 the others
    const uint32_t lanes = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const int t = (warp & 3) * 32 + lane, half = warp >> 2;
    bool ok = mbar_wait(&bars[DO_S], 0, abort_word);
    tc_fence_after();
    __syncwarp();
    {
      uint32_t hi[32], lo[32];
#pragma unroll
      for (int c0 = 0; c0 < 64; c0 += 32) {
        uint32_t r[32];
        const int col = half * 64 + c0;
        tmem_ld_32x32b_x32(t_s + lanes + col, r);
        tmem_ld_wait();
#pragma unroll
        for (int e = 0; e < 32; e += 2) {
          const int d = t - (col + e);  // tokens between the key and this row
          const float x = d >= 0 ? __uint_as_float(r[e]) * pw[d] : 0.f;
          const float y = d >= 1 ? __uint_as_float(r[e + 1]) * pw[d - 1] : 0.f;
          split_pair(x, y, hi[(c0 + e) >> 1], lo[(c0 + e) >> 1]);
        }
      }
      tc_fence_before();
      workers_sync();  // (both halves of the row have been read)
      tc_fence_after();
      tmem_st_32x32b_x32(t_hi + lanes + half * 32, hi);
      tmem_st_32x32b_x32(t_lo + lanes + half * 32, lo);
      tmem_st_wait();
    }
    uint32_t cr[2][32];
    if (carried) {
      ok = ok && mbar_wait(&bars[DO_C], 0, abort_word);
      __syncwarp();
      tc_fence_after();
      tmem_ld_32x32b_x32(t_o + lanes + half * 64, cr[0]);
      tmem_ld_32x32b_x32(t_o + lanes + half * 64 + 32, cr[1]);
      tmem_ld_wait();
    } else {
#pragma unroll
      for (int e = 0; e < 32; ++e) cr[0][e] = cr[1][e] = 0u;
    }
    tc_fence_before();
    __syncwarp();
    if (lane == 0 && ok) mbar_arrive(&bars[DO_P]);
    ok = mbar_wait(&bars[DO_O], 0, abort_word);
    __syncwarp();
    tc_fence_after();
    const float f = pw[t + 1];
#pragma unroll
    for (int i = 0; i < 2; ++i) {  // into Q's place, in the store's 128-byte swizzle
      uint32_t r[32];
      tmem_ld_32x32b_x32(t_o + lanes + half * 64 + i * 32, r);
      tmem_ld_wait();
#pragma unroll
      for (int e = 0; e < 32; e += 8) {
        float v[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) v[k] = fmaf(f, __uint_as_float(cr[i][e + k]), __uint_as_float(r[e + k]));
        const int j = i * 4 + (e >> 3);
        Vec8<uint16_t>::store(reinterpret_cast<uint16_t*>(q_s + half * DC_BOX + t * 128 + ((j ^ (t & 7)) << 4)), v);
      }
    }
    fence_proxy_async_smem();
    workers_sync();
    if (threadIdx.x == 0 && ok && *abort_word == 0) {  // (rows behind the input's end are not stored)
      tma_store_4d(&tmO, q_s, 0, c * DC, h, b);
      tma_store_4d(&tmO, q_s + DC_BOX, 64, c * DC, h, b);
      tma_store_commit();
      tma_store_wait_all<0>();
    }
    __syncwarp();
  }
  tc_fence_before();
  __syncthreads();
  if (warp == DO_WORKERS / 32) {
    tc_fence_after();
    tmem_dealloc(t_s, 256);
  }
  if (threadIdx.x == 0 && abort_flag) atomicExch(p.status, YTC_TIMEOUT);
}

static bool chunks_allowed(const DecayedAttn& a) {
  auto aligned = [](const void* p) { return (reinterpret_cast<uint64_t>(p) & 15u) == 0; };
  return a.dtype == YTC_BF16 && a.dim == DC && a.vdim == DC && a.ld % 8 == 0 && a.ld_o % 8 == 0 && !a.pos && aligned(a.q) &&
         aligned(a.k) && aligned(a.v) && aligned(a.o);
}

static int token_map(CUtensorMap* m, const void* base, int64_t ld, const DecayedAttn& a, int batch) {
  // {column, token, head, sequence}
  const uint64_t dims[4] = {DC, static_cast<uint64_t>(a.len), static_cast<uint64_t>(a.heads), static_cast<uint64_t>(batch)};
  const uint64_t strides[3] = {static_cast<uint64_t>(ld) * 2, DC * 2, static_cast<uint64_t>(ld) * a.len * 2};
  const uint32_t box[4] = {64, DC, 1, 1};
  return encode_tensor_map(m, CU_TENSOR_MAP_DATA_TYPE_UINT16, 4, base, dims, strides, box, CU_TENSOR_MAP_SWIZZLE_128B);
}

static int decayed_chunks(const DecayedAttn& all, cudaStream_t st) {
  const int chunks = (all.len + DC - 1) / DC;
  const int64_t per_seq = static_cast<int64_t>(all.heads) * chunks;  // units
  const int64_t unit_bytes = DC_STATE * 8;
  // as many sequences at a time as fit the scratch memory that stays allocated
  const int group = static_cast<int>(std::max<int64_t>(1, std::min<int64_t>(all.batch, (256ll << 20) / (per_seq * unit_bytes))));
  int* status = device_status_word();
  if (!status) {
    set_last_error("decayed_attention: no device status word");
    return YTC_CUDA_ERROR;
  }
  YTC_REQUIRE(group * per_seq * 2 * DC <= 0x7fffffffll, "decayed_attention: too many chunks");
  int s = ensure_dynamic_smem(reinterpret_cast<const void*>(decayed_chunk_state_kernel), DS_SMEM);
  if (s == YTC_OK) s = ensure_dynamic_smem(reinterpret_cast<const void*>(decayed_chunk_out_kernel), DO_SMEM);
  if (s != YTC_OK) return s;
  auto* ws = static_cast<char*>(device_workspace(static_cast<size_t>(group * per_seq * unit_bytes), st));
  if (!ws) {
    set_last_error("decayed_attention: no scratch memory");
    return YTC_CUDA_ERROR;
  }
  for (int b0 = 0; b0 < all.batch; b0 += group) {
    DecayedAttn a = all;
    const int nb = std::min(group, all.batch - b0);
    const int64_t in_off = static_cast<int64_t>(b0) * a.len * a.ld * 2;
    a.q = static_cast<const char*>(a.q) + in_off;
    a.k = static_cast<const char*>(a.k) + in_off;
    a.v = static_cast<const char*>(a.v) + in_off;
    DecayedChunks p;
    p.own = reinterpret_cast<float*>(ws);
    p.planes = reinterpret_cast<uint16_t*>(ws + group * per_seq * DC_STATE * 4);
    p.decay = a.decay;
    p.state = a.state + b0 * static_cast<int64_t>(a.heads) * DC_STATE;
    a.o = static_cast<char*>(a.o) + static_cast<int64_t>(b0) * a.len * a.ld_o * 2;
    p.heads = a.heads; p.chunks = chunks; p.len = a.len; p.first = a.first ? 1 : 0;
    p.status = status;
    CUtensorMap tmQ, tmK, tmV, tmO, tmU, tmS;
    if ((s = token_map(&tmQ, a.q, a.ld, a, nb)) != YTC_OK) return s;
    if ((s = token_map(&tmK, a.k, a.ld, a, nb)) != YTC_OK) return s;
    if ((s = token_map(&tmV, a.v, a.ld, a, nb)) != YTC_OK) return s;
    if ((s = token_map(&tmO, a.o, a.ld_o, a, nb)) != YTC_OK) return s;
    {
      const uint64_t rows = static_cast<uint64_t>(nb * per_seq) * DC;
      const uint64_t dims_u[2] = {DC, rows}, strides_u[1] = {DC * 4}, dims_s[2] = {DC, 2 * rows}, strides_s[1] = {DC * 2};
      const uint32_t box_u[2] = {32, DC}, box_s[2] = {64, DC};
      s = encode_tensor_map(&tmU, CU_TENSOR_MAP_DATA_TYPE_FLOAT32, 2, p.own, dims_u, strides_u, box_u, CU_TENSOR_MAP_SWIZZLE_128B);
      if (s != YTC_OK) return s;
      s = encode_tensor_map(&tmS, CU_TENSOR_MAP_DATA_TYPE_UINT16, 2, p.planes, dims_s, strides_s, box_s, CU_TENSOR_MAP_SWIZZLE_128B);
      if (s != YTC_OK) return s;
    }
    const dim3 grid(chunks, a.heads, nb);
    YTC_CUDA(launch_overlapped(decayed_chunk_state_kernel, grid, dim3(DS_THREADS), DS_SMEM, st, tmK, tmV, tmU, p));
    YTC_CUDA(launch_overlapped(decayed_chunk_scan_kernel, dim3(DC_STATE / 4 / DN_THREADS, a.heads, nb), dim3(DN_THREADS), 0, st, p));
    YTC_CUDA(launch_overlapped(decayed_chunk_out_kernel, grid, dim3(DO_THREADS), DO_SMEM, st, tmQ, tmK, tmV, tmS, tmO, p));
    count_launch(3);
    YTC_CUDA(cudaGetLastError());
  }
  device_workspace_release(st);
  return YTC_OK;
}

constexpr int DC_MIN_TOKENS = 48;  // below, the token-by-token kernel is faster than three launches

int decayed_attention(const DecayedAttn& a, cudaStream_t st) {
  if (a.len <= 0 || a.batch <= 0) return YTC_OK;
  YTC_REQUIRE(a.heads > 0 && a.dim > 0 && a.dim % 8 == 0 && a.vdim > 0 && a.vdim % 8 == 0 && (!a.pos || a.len == 1) &&
                  a.heads <= 65535 && a.batch <= 65535,
              "decayed_attention: bad extent");
  const bool allowed = chunks_allowed(a);
  if (a.path == 2 && !allowed) {
    set_last_error("decayed_attention: chunks want bf16 heads of %d x %d", DC, DC);
    return YTC_UNSUPPORTED;
  }
  if (a.path == 2 || (a.path == 0 && allowed && a.len >= DC_MIN_TOKENS)) return decayed_chunks(a, st);
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
