// One new token of a language model: the kernels of a decode step that the models share.
//
// A step is a chain of short kernels (projection with the norms before it, attention, projection, ...) queued as
// programmatic dependent launches inside a CUDA graph. Every kernel requests what does not depend on the kernel in
// front of it (the weights it will multiply by, norm weights, the residual row, old keys and values) BEFORE it waits for
// that kernel, so that the weight stream does not stop at kernel boundaries. A kernel lets the next one start once it
// has passed its own wait: at most two kernels of the chain run at a time, and what a kernel reads before its wait was
// written at least two kernels earlier. Activations are fp32 vectors of a few KB; every CTA stages the whole vector in
// shared memory and recomputes the norms from it, which costs less than one more hand-over. Loops are kept rolled:
// a kernel of this chain runs its code once, at the speed the instructions arrive.
#include <math_constants.h>

#include "lm_ops.cuh"

namespace ytk {

constexpr int DL_THREADS = 512, DL_WARPS = DL_THREADS / 32;
constexpr int DL_PIECE = 256;              // columns a warp covers with one 16-byte load per lane
constexpr int DL_DEPTH = 4;                // row-pair pieces in flight per warp
constexpr int DL_RING = DL_DEPTH * 2 * 512;  // bytes of a warp's weight ring

// ---------------------------------------------------------------- asynchronous copies of 16 bytes per lane
__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))),
               "l"(src)
               : "memory");
}
__device__ __forceinline__ void cp_async16_or_zero(void* dst, const void* src, bool ok) {
  const int bytes = ok ? 16 : 0;  // (0: the 16 bytes are zero-filled, nothing is read)
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))),
               "l"(src), "r"(bytes)
               : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

__device__ __forceinline__ float dl_block_sum(float v, float* red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < DL_WARPS; ++i) t += red[i];
  return t;
}

// ---------------------------------------------------------------- the staged input vector
// Element c of the vector stands where the lane that multiplies it reads 16 bytes without bank conflicts: a piece of
// 256 is 32 lanes x 8 elements, first the lanes' elements 0 .. 3, then 4 .. 7.
__device__ __forceinline__ int staged_at(int c) { return (c & ~255) + ((c & 4) << 5) + ((c & 255) >> 3) * 4 + (c & 3); }

struct InputSmem {  // shared memory of a staged input
  float* h;         // [padded] the vector, in staged order
  float *x, *g_post, *g_pre;  // [k] residual row and norm weights (DECODE_GATED: g_post is the gate, no x)
};
__host__ __device__ __forceinline__ int input_floats(int kind, int k, int padded) {
  return padded + (kind == DECODE_PLAIN ? 0 : kind == DECODE_GATED ? 2 * k : 3 * k);
}
__device__ __forceinline__ InputSmem input_smem(int kind, float* p, int k, int padded) {
  if (kind == DECODE_GATED) return InputSmem{p, nullptr, p + padded, p + padded + k};
  return InputSmem{p, p + padded, p + padded + k, p + padded + 2 * k};
}

// Requests what the input needs besides the output of the kernel before (one copy group).
__device__ __forceinline__ void prefetch_input(const DecodeInput& in, int k, const InputSmem& s) {
  if (in.kind != DECODE_PLAIN)
    for (int c = threadIdx.x * 4; c < k; c += DL_THREADS * 4) {
      if (in.w_pre) cp_async16(s.g_pre + c, in.w_pre + c);
      if (in.kind == DECODE_RESIDUAL) {
        cp_async16(s.g_post + c, in.w_post + c);
        cp_async16(s.x + c, in.x_in + c);
      }
      if (in.kind == DECODE_GATED && in.gate) cp_async16(s.g_post + c, in.gate + c);  // (written two kernels ago)
    }
  cp_async_commit();
}

// After the wait. `older`: copy groups issued after prefetch_input that may still be in flight. `writer`: this CTA
// stores the new residual row (and the normed vector, when h_out is given).
template <int OLDER>
__device__ __forceinline__ void stage_input(const DecodeInput& in, int k, int padded, const InputSmem& s, float* red,
                                            bool writer, float* h_out) {
  for (int c = k + threadIdx.x * 4; c < padded; c += DL_THREADS * 4)
    *reinterpret_cast<float4*>(s.h + staged_at(c)) = make_float4(0.f, 0.f, 0.f, 0.f);
  if (in.kind == DECODE_PLAIN) {
    for (int c = threadIdx.x * 4; c < k; c += DL_THREADS * 4)
      *reinterpret_cast<float4*>(s.h + staged_at(c)) = *reinterpret_cast<const float4*>(in.plain + c);
    __syncthreads();
    return;
  }
  float ss = 0.f;
  if (in.kind == DECODE_GATED) {
    for (int c = threadIdx.x * 4; c < k; c += DL_THREADS * 4) {
      const float4 v = *reinterpret_cast<const float4*>(in.plain + c);
      *reinterpret_cast<float4*>(s.h + staged_at(c)) = v;
      ss = fmaf(v.x, v.x, ss); ss = fmaf(v.y, v.y, ss); ss = fmaf(v.z, v.z, ss); ss = fmaf(v.w, v.w, ss);
    }
    const float inv = in.w_pre ? 1.0f / sqrtf(dl_block_sum(ss, red) / in.width + in.eps) : 1.f;
    cp_async_wait<OLDER>();
    for (int c = threadIdx.x * 4; c < k; c += DL_THREADS * 4) {
      float4 v = *reinterpret_cast<const float4*>(s.h + staged_at(c));
      if (in.w_pre) {
        const float4 g = *reinterpret_cast<const float4*>(s.g_pre + c);
        v.x *= inv * g.x; v.y *= inv * g.y; v.z *= inv * g.z; v.w *= inv * g.w;
      }
      if (in.gate) {
        const float4 g = *reinterpret_cast<const float4*>(s.g_post + c);
        v.x *= lm_sigmoid(g.x); v.y *= lm_sigmoid(g.y); v.z *= lm_sigmoid(g.z); v.w *= lm_sigmoid(g.w);
      }
      *reinterpret_cast<float4*>(s.h + staged_at(c)) = v;
    }
    __syncthreads();
    return;
  }
  if (in.kind == DECODE_EMBED) {
    int id = *in.id;
    id = id < 0 ? 0 : (id >= in.vocab ? in.vocab - 1 : id);
    const uint16_t* row = in.embed + static_cast<int64_t>(id) * k;
    for (int c = threadIdx.x * 4; c < k; c += DL_THREADS * 4) {
      const uint2 u = *reinterpret_cast<const uint2*>(row + c);
      const float e = in.embed_scale;
      const float4 x = make_float4(e * __uint_as_float(u.x << 16), e * __uint_as_float(u.x & 0xFFFF0000u),
                                   e * __uint_as_float(u.y << 16), e * __uint_as_float(u.y & 0xFFFF0000u));
      *reinterpret_cast<float4*>(s.x + c) = x;  // (every thread reads back its own columns only)
      if (writer) *reinterpret_cast<float4*>(in.x_out + c) = x;
    }
    cp_async_wait<OLDER>();
  } else {
    for (int c = threadIdx.x * 4; c < k; c += DL_THREADS * 4) {
      const float4 y = *reinterpret_cast<const float4*>(in.y + c);
      *reinterpret_cast<float4*>(s.h + staged_at(c)) = y;
      ss = fmaf(y.x, y.x, ss); ss = fmaf(y.y, y.y, ss); ss = fmaf(y.z, y.z, ss); ss = fmaf(y.w, y.w, ss);
    }
    const float inv = 1.0f / sqrtf(dl_block_sum(ss, red) / in.width + in.eps);
    cp_async_wait<OLDER>();
    for (int c = threadIdx.x * 4; c < k; c += DL_THREADS * 4) {
      const float4 y = *reinterpret_cast<const float4*>(s.h + staged_at(c)), g = *reinterpret_cast<const float4*>(s.g_post + c);
      float4 x = *reinterpret_cast<const float4*>(s.x + c);
      x.x += y.x * inv * g.x; x.y += y.y * inv * g.y; x.z += y.z * inv * g.z; x.w += y.w * inv * g.w;
      *reinterpret_cast<float4*>(s.x + c) = x;
      if (writer) *reinterpret_cast<float4*>(in.x_out + c) = x;
    }
  }
  if (!in.w_pre) {
    for (int c = threadIdx.x * 4; c < k; c += DL_THREADS * 4) {
      const float4 x = *reinterpret_cast<const float4*>(s.x + c);
      *reinterpret_cast<float4*>(s.h + staged_at(c)) = x;
      if (writer && h_out) *reinterpret_cast<float4*>(h_out + c) = x;
    }
    __syncthreads();
    return;
  }
  ss = 0.f;
  for (int c = threadIdx.x * 4; c < k; c += DL_THREADS * 4) {
    const float4 x = *reinterpret_cast<const float4*>(s.x + c);
    ss = fmaf(x.x, x.x, ss); ss = fmaf(x.y, x.y, ss); ss = fmaf(x.z, x.z, ss); ss = fmaf(x.w, x.w, ss);
  }
  const float inv = 1.0f / sqrtf(dl_block_sum(ss, red + DL_WARPS) / in.width + in.eps);
  for (int c = threadIdx.x * 4; c < k; c += DL_THREADS * 4) {
    const float4 g = *reinterpret_cast<const float4*>(s.g_pre + c);
    float4 x = *reinterpret_cast<const float4*>(s.x + c);
    x.x *= inv * g.x; x.y *= inv * g.y; x.z *= inv * g.z; x.w *= inv * g.w;
    *reinterpret_cast<float4*>(s.h + staged_at(c)) = x;
    if (writer && h_out) *reinterpret_cast<float4*>(h_out + c) = x;
  }
  __syncthreads();
}

// ---------------------------------------------------------------- products of weight rows with the staged vector
// A CTA owns output row pairs [begin, end); `ks` warps share a pair and split its pieces of 256 columns. Every lane
// copies its own 16 bytes of both rows of a piece into the warp's ring in shared memory and reads them back itself:
// DL_DEPTH pieces are in flight, no barrier is involved, and the loop stays rolled. addr(pair, piece, &row0, &row1, &ok)
// gives the lane's addresses (ok: inside the row). Partial sums go to part[((pair - begin) * 2 + r) * ks + sub].
template <typename Addr>
struct RowPairs {
  Addr addr;
  uint8_t* ring;
  int end, pieces, ks, sub, slots, begin;
  int lp, lpc, ls = 0;  // next piece to request: pair, piece, ring slot
  __device__ RowPairs(Addr f, uint8_t* rings, int begin_, int end_, int pieces_, int ks_)
      : addr(f), end(end_), pieces(pieces_), ks(ks_), begin(begin_) {
    const int warp = threadIdx.x >> 5;
    ring = rings + warp * DL_RING + (threadIdx.x & 31) * 16;
    sub = warp % ks;
    slots = DL_WARPS / ks;
    lp = begin + warp / ks;
    lpc = sub;
  }
  __device__ __forceinline__ void request() {  // one copy group, empty past the end
    if (lp < end) {
      const uint16_t *p0, *p1;
      bool ok0, ok1;
      addr(lp, lpc, p0, p1, ok0, ok1);
      cp_async16_or_zero(ring + ls * 1024, p0, ok0);
      cp_async16_or_zero(ring + ls * 1024 + 512, p1, ok1);
      lpc += ks;
      if (lpc >= pieces) {
        lpc = sub;
        lp += slots;
      }
    }
    cp_async_commit();
    ls = (ls + 1) & (DL_DEPTH - 1);
  }
  __device__ __forceinline__ void start() {  // DL_DEPTH - 1 groups
#pragma unroll 1
    for (int i = 0; i < DL_DEPTH - 1; ++i) request();
  }
  // h: the staged vector, piece p at h + 256 p
  __device__ __forceinline__ void run(const float* h, float* part) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    int slot = 0;
#pragma unroll 1
    for (int pair = begin + warp / ks; pair < end; pair += slots) {
      float a0 = 0.f, a1 = 0.f;
#pragma unroll 1
      for (int piece = sub; piece < pieces; piece += ks) {
        request();
        cp_async_wait<DL_DEPTH - 1>();
        const uint4 w0 = *reinterpret_cast<const uint4*>(ring + slot * 1024);
        const uint4 w1 = *reinterpret_cast<const uint4*>(ring + slot * 1024 + 512);
        slot = (slot + 1) & (DL_DEPTH - 1);
        const float4 xa = *reinterpret_cast<const float4*>(h + piece * DL_PIECE + lane * 4);
        const float4 xb = *reinterpret_cast<const float4*>(h + piece * DL_PIECE + 128 + lane * 4);
        const float x[8] = {xa.x, xa.y, xa.z, xa.w, xb.x, xb.y, xb.z, xb.w};
        float w[8];
        Vec8<uint16_t>::unpack(w0, w);
#pragma unroll
        for (int e = 0; e < 8; ++e) a0 = fmaf(x[e], w[e], a0);
        Vec8<uint16_t>::unpack(w1, w);
#pragma unroll
        for (int e = 0; e < 8; ++e) a1 = fmaf(x[e], w[e], a1);
      }
      // both sums at once: the lower half of the warp finishes row 0, the upper half row 1
      const float other = __shfl_xor_sync(0xffffffffu, lane < 16 ? a1 : a0, 16);
      float v = (lane < 16 ? a0 : a1) + other;
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
      if ((lane & 15) == 0) part[((pair - begin) * 2 + (lane >> 4)) * ks + sub] = v;
    }
  }
};

__device__ __forceinline__ float sum_sub(const float* part, int row, int ks) {
  float s = 0.f;
  for (int i = 0; i < ks; ++i) s += part[row * ks + i];
  return s;
}

// Warps that share a row pair: the count with the fewest pieces per warp.
static int pick_ks(int pairs_per_cta, int pieces) {
  int best = 1;
  double best_cost = 1e30;
  for (int ks = 1; ks <= DL_WARPS && ks <= pieces; ks *= 2) {
    const int slots = DL_WARPS / ks;
    const double rounds = (pairs_per_cta + slots - 1) / slots;
    const double cost = rounds * ((pieces + ks - 1) / ks + 2);  // (the sum over the lanes costs about two pieces)
    if (cost < best_cost * 0.95) {
      best_cost = cost;
      best = ks;
    }
  }
  return best;
}

__device__ __forceinline__ void my_pairs(int pairs, int& begin, int& end) {
  begin = static_cast<int>(static_cast<int64_t>(pairs) * blockIdx.x / gridDim.x);
  end = static_cast<int>(static_cast<int64_t>(pairs) * (blockIdx.x + 1) / gridDim.x);
}

static int dl_smem_check(const void* fn, int smem, const char* what) {
  if (smem > 220 * 1024) {
    set_last_error("decode step: %s does not fit shared memory (%d bytes)", what, smem);
    return YTC_UNSUPPORTED;
  }
  return smem > 48 * 1024 ? ensure_dynamic_smem(fn, smem) : YTC_OK;
}
static int check_input(const DecodeInput& in, int k) {
  YTC_REQUIRE(k > 0 && k % 8 == 0 && (in.kind == DECODE_PLAIN || in.width <= k), "decode step: bad vector length %d", k);
  return YTC_OK;
}

// ------------------------------------------------------------------ linear
__global__ void __launch_bounds__(DL_THREADS, 2) decode_linear_kernel(const DecodeLinear p, int ks, int padded) {
  extern __shared__ __align__(16) uint8_t dl_smem[];  // weight rings, input, part[]
  __shared__ float red[2 * DL_WARPS];
  const InputSmem in = input_smem(p.in.kind, reinterpret_cast<float*>(dl_smem + DL_WARPS * DL_RING), p.k, padded);
  float* part = in.h + input_floats(p.in.kind, p.k, padded);
  int begin, end;
  my_pairs((p.n + 1) / 2, begin, end);
  const int lane8 = (threadIdx.x & 31) * 8;
  auto addr = [&](int pair, int piece, const uint16_t*& p0, const uint16_t*& p1, bool& ok0, bool& ok1) {
    const int col = piece * DL_PIECE + lane8;
    ok0 = col < p.k;
    ok1 = ok0 && 2 * pair + 1 < p.n;
    p0 = p.w + static_cast<int64_t>(2 * pair) * p.k + (ok0 ? col : 0);
    p1 = ok1 ? p0 + p.k : p0;
  };
  RowPairs<decltype(addr)> rp(addr, dl_smem, begin, end, (p.k + DL_PIECE - 1) / DL_PIECE, ks);
  prefetch_input(p.in, p.k, in);
  rp.start();
  dependent_wait();
  dependent_trigger();
  stage_input<DL_DEPTH - 1>(p.in, p.k, padded, in, red, blockIdx.x == 0, nullptr);
  rp.run(in.h, part);
  __syncthreads();
  for (int i = threadIdx.x; i < (end - begin) * 2; i += DL_THREADS) {
    const int row = begin * 2 + i;
    if (row >= p.n) continue;
    p.out[row] = lm_activation(p.ex, sum_sub(part, i, ks), row);
  }
  if (p.advance && blockIdx.x == 0 && threadIdx.x == 0) *p.advance += 1;
}

int decode_linear(const DecodeLinear& a, cudaStream_t st) {
  int s = check_input(a.in, a.k);
  if (s != YTC_OK) return s;
  const int pieces = (a.k + DL_PIECE - 1) / DL_PIECE, padded = pieces * DL_PIECE, pairs = (a.n + 1) / 2;
  const int grid = pairs < sm_count() ? pairs : sm_count();
  const int per = (pairs + grid - 1) / grid;
  const int ks = pick_ks(per, pieces);
  const int smem = DL_WARPS * DL_RING + (input_floats(a.in.kind, a.k, padded) + per * 2 * ks) * static_cast<int>(sizeof(float));
  if ((s = dl_smem_check(reinterpret_cast<const void*>(decode_linear_kernel), smem, "a projection")) != YTC_OK) return s;
  YTC_CUDA(launch_overlapped(decode_linear_kernel, dim3(grid), dim3(DL_THREADS), smem, st, a, ks, padded));
  count_launch();
  YTC_CUDA(cudaGetLastError());
  return YTC_OK;
}

// ------------------------------------------------------------------ attention
// One cluster of CTAs per K/V head and block of one, two or four query heads of its group; the keys of the window are
// split over all warps of the cluster. A warp works on its own: it copies DA_KW keys and values at a time into its part of
// shared memory (the first ones requested before the wait for the projection), takes the scores with eight lanes per
// key, and sums the values with the value dim across its lanes. Warps meet through shared memory; the CTAs push their
// results into the shared memory of the cluster's first CTA, which adds them.
constexpr int DA_MAX_CLUSTER = 8;
template <typename T>
constexpr int DA_KW = sizeof(T) == 2 ? 8 : 4;  // keys per step of a warp

__device__ __forceinline__ void cluster_barrier() {
  asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
  asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}
template <typename T>
__device__ __forceinline__ void load4(const T* p, float (&f)[4]) {
  if (sizeof(T) == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  } else {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    f[0] = __uint_as_float(u.x << 16); f[1] = __uint_as_float(u.x & 0xFFFF0000u);
    f[2] = __uint_as_float(u.y << 16); f[3] = __uint_as_float(u.y & 0xFFFF0000u);
  }
}

// Stores to the shared memory of CTA `rank` of the cluster.
__device__ __forceinline__ void st_cluster(float* p, uint32_t rank, float v) {
  uint32_t a = static_cast<uint32_t>(__cvta_generic_to_shared(p)), r;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(a), "r"(rank));
  asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(r), "f"(v) : "memory");
}

// NH: query heads per cluster, NV: float4 slots of the value dim per lane (1: up to 128, 2: up to 256).
template <typename T, int NH, int NV>
__global__ void __launch_bounds__(DL_THREADS, NV == 1 ? 2 : 1) decode_attn_kernel(const DecodeAttn p, int ncta, int nbuf) {
  constexpr int KW = DA_KW<T>;
  // K/V of the warps [warps][nbuf][KW][dim + vdim] (T), q[NH][dim], o[warps][NH][vdim], the CTAs' results
  // x[cluster][NH][vdim] (in CTA 0)
  extern __shared__ __align__(16) uint8_t da_smem[];
  __shared__ float w_s[DL_WARPS][NH][KW], al_s[DL_WARPS][NH], m_s[DL_WARPS][NH], l_s[DL_WARPS][NH];
  __shared__ float xm[DA_MAX_CLUSTER][NH], xl[DA_MAX_CLUSTER][NH];
  const int D = p.dim, Dv = p.vdim, row_e = D + Dv;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  T* kv_s = reinterpret_cast<T*>(da_smem) + static_cast<size_t>(warp) * nbuf * KW * row_e;
  float* q_s = reinterpret_cast<float*>(da_smem + static_cast<size_t>(DL_WARPS) * nbuf * KW * row_e * sizeof(T));
  float* o_s = q_s + NH * D;
  float* x_s = o_s + (DL_WARPS * NH * Dv > row_e ? DL_WARPS * NH * Dv : row_e);
  const int unit = blockIdx.x / ncta, rank = blockIdx.x - unit * ncta;
  const int blocks = (p.groups + NH - 1) / NH;
  const int g = unit / blocks, h0 = (unit - g * blocks) * NH;  // K/V head, first query head of the group
  const int nh = p.groups - h0 < NH ? p.groups - h0 : NH;
  if (ncta > 1) asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");  // (this CTA has started)

  // (the position word was written before this step's first kernel started)
  const int pos = *p.pos;
  const int seen = (p.window > 0 && pos + 1 > p.window) ? p.window : pos + 1;
  const int old_n = seen - 1;  // positions pos - old_n .. pos - 1, then the new one
  const int warps = ncta * DL_WARPS, wi = rank * DL_WARPS + warp;
  const int per = (old_n + warps - 1) / warps;
  const int k0 = wi * per < old_n ? wi * per : old_n;
  const int k1 = k0 + per < old_n ? k0 + per : old_n;
  const bool has_new = wi == warps - 1;  // the last warp (the one with the fewest old keys) takes the new key
  const int mine = k1 - k0 + (has_new ? 1 : 0);
  const T* kr = static_cast<const T*>(p.k) + static_cast<int64_t>(g) * p.ring * D;
  const T* vr = static_cast<const T*>(p.v) + static_cast<int64_t>(g) * p.ring * Dv;
  const int row0 = (pos - old_n + k0) % p.ring;
  constexpr int VE = 16 / sizeof(T);  // elements per 16 bytes
  const int kp = D / VE, vp = Dv / VE;
  auto fetch = [&](int c0, int buf) {  // requests old keys c0 .. of this warp (one copy group)
    T* dst = kv_s + buf * KW * row_e;
    const int n = (k1 - k0) - c0 < KW ? (k1 - k0) - c0 : KW;
    int row = row0 + c0;
#pragma unroll 1
    for (int key = 0; key < n; ++key, ++row) {
      const int64_t r = row >= p.ring ? row - p.ring : row;
      for (int c = lane; c < kp + vp; c += 32)
        cp_async16(dst + key * row_e + c * VE, c < kp ? kr + r * D + c * VE : vr + r * Dv + (c - kp) * VE);
    }
    cp_async_commit();
  };
  fetch(0, 0);
  if (nbuf > 1) fetch(KW, 1);
  const float lam = p.mix == VMIX_MIX ? *p.lambda : 0.f;
  dependent_wait();
  dependent_trigger();
  const int H = p.kv_heads * p.groups;
  for (int i = threadIdx.x * 4; i < nh * D; i += DL_THREADS * 4)
    *reinterpret_cast<float4*>(q_s + i) =
        *reinterpret_cast<const float4*>(p.qkv + static_cast<int64_t>(g * p.groups + h0) * D + i);
  if (has_new) {  // the new key and value: behind the warp's old keys, and (one cluster per K/V head) into the rings
    const float* k_new = p.qkv + static_cast<int64_t>(H) * D + static_cast<int64_t>(g) * D;
    const float* v_new = p.qkv + static_cast<int64_t>(H + p.kv_heads) * D + static_cast<int64_t>(g) * Dv;
    const int64_t row = pos % p.ring;
    T* kw = static_cast<T*>(p.k) + (static_cast<int64_t>(g) * p.ring + row) * D;
    T* vw = static_cast<T*>(p.v) + (static_cast<int64_t>(g) * p.ring + row) * Dv;
    const bool first_block = h0 == 0;
    for (int i = lane; i < (D + Dv) / 8; i += 32) {
      float f[8];
      const int e = i * 8;
      if (e < D) {
        Vec8<float>::load(k_new + e, f);
      } else {
        float* first = p.v_first + static_cast<int64_t>(g) * Dv + e - D;
        Vec8<float>::load(v_new + e - D, f);
        if (p.mix == VMIX_FIRST && first_block) Vec8<float>::store(first, f);
        if (p.mix == VMIX_MIX) {
          float v0[8];
          Vec8<float>::load(first, v0);
#pragma unroll
          for (int k = 0; k < 8; ++k) f[k] = (1.f - lam) * f[k] + lam * v0[k];
        }
      }
      if (first_block) Vec8<T>::store(e < D ? kw + e : vw + e - D, f);
      Vec8<float>::store(o_s + e, f);  // joins the keys in shared memory when their last step is reached
    }
  }
  if (lane < NH) {
    m_s[warp][lane] = -CUDART_INF_F;
    l_s[warp][lane] = 0.f;
  }
  __syncthreads();
  float acc[NH][NV * 4] = {};
#pragma unroll 1
  for (int c0 = 0, buf = 0; c0 < mine; c0 += KW, buf = (buf + 1 == nbuf ? 0 : buf + 1)) {
    const int n = mine - c0 < KW ? mine - c0 : KW;
    if (nbuf > 1) cp_async_wait<1>();
    else cp_async_wait<0>();
    T* kv = kv_s + buf * KW * row_e;
    if (has_new && c0 + n == mine) {
      for (int i = lane; i < row_e / 8; i += 32) {
        float f[8];
        Vec8<float>::load(o_s + i * 8, f);
        Vec8<T>::store(kv + (n - 1) * row_e + i * 8, f);
      }
    }
    __syncwarp();
    // scores: eight lanes per key, four keys at a time
#pragma unroll 1
    for (int key0 = 0; key0 < n; key0 += 4) {
      const int key = key0 + (lane >> 3);
      const T* k = kv + (key < n ? key : 0) * row_e;
      float dot[NH] = {};
      for (int c = (lane & 7) * 8; c < D; c += 64) {
        float a[8];
        Vec8<T>::load(k + c, a);
#pragma unroll
        for (int h = 0; h < NH; ++h) {
          if (h >= nh) break;
          float b[8];
          Vec8<float>::load(q_s + h * D + c, b);
#pragma unroll
          for (int e = 0; e < 8; ++e) dot[h] = fmaf(a[e], b[e], dot[h]);
        }
      }
#pragma unroll
      for (int h = 0; h < NH; ++h) {
        dot[h] += __shfl_xor_sync(0xffffffffu, dot[h], 1);
        dot[h] += __shfl_xor_sync(0xffffffffu, dot[h], 2);
        dot[h] += __shfl_xor_sync(0xffffffffu, dot[h], 4);
        if ((lane & 7) == 0 && key < n) w_s[warp][h][key] = dot[h] * p.scale;
      }
    }
    __syncwarp();
    // weights: KW lanes per head
#pragma unroll 1
    for (int hb = 0; hb < nh; hb += 32 / KW) {
      const int h = hb + lane / KW, key = lane % KW;
      const int hc = h < nh ? h : 0;
      float s = -CUDART_INF_F;
      if (h < nh && key < n) {
        s = w_s[warp][h][key];
        if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
      }
      float m = s;
#pragma unroll
      for (int o = KW / 2; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
      const float m_old = m_s[warp][hc], m_new = fmaxf(m_old, m);
      const float w = s == -CUDART_INF_F ? 0.f : expf(s - m_new);
      float l = w;
#pragma unroll
      for (int o = KW / 2; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
      __syncwarp();
      if (h < nh) {
        w_s[warp][h][key] = w;
        if (key == 0) {
          const float alpha = m_old == -CUDART_INF_F ? 0.f : expf(m_old - m_new);
          al_s[warp][h] = alpha;
          m_s[warp][h] = m_new;
          l_s[warp][h] = l_s[warp][h] * alpha + l;
        }
      }
    }
    __syncwarp();
#pragma unroll
    for (int h = 0; h < NH; ++h) {
      const float alpha = h < nh ? al_s[warp][h] : 0.f;
#pragma unroll
      for (int e = 0; e < NV * 4; ++e) acc[h][e] *= alpha;
    }
#pragma unroll 2
    for (int key = 0; key < n; ++key) {
      float v[NV][4] = {};
#pragma unroll
      for (int j = 0; j < NV; ++j)
        if (j * 128 + lane * 4 < Dv) load4<T>(kv + key * row_e + D + j * 128 + lane * 4, v[j]);
#pragma unroll
      for (int h = 0; h < NH; ++h) {
        const float w = h < nh ? w_s[warp][h][key] : 0.f;
#pragma unroll
        for (int e = 0; e < NV * 4; ++e) acc[h][e] = fmaf(w, v[e >> 2][e & 3], acc[h][e]);
      }
    }
    __syncwarp();
    if (c0 + nbuf * KW < mine) fetch(c0 + nbuf * KW, buf);
    else cp_async_commit();
  }
  __syncthreads();  // (the new key's copy in o_s has been read)
  // The CTA's result: the warps' sums, brought to the CTA's maximum by every warp itself.
  float mc[NH];
#pragma unroll
  for (int h = 0; h < NH; ++h) {
    float m = lane < DL_WARPS ? m_s[lane][h] : -CUDART_INF_F;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
    mc[h] = m;
    const float f = m_s[warp][h] == -CUDART_INF_F ? 0.f : expf(m_s[warp][h] - m);
#pragma unroll
    for (int j = 0; j < NV; ++j)
      if (j * 128 + lane * 4 < Dv)
        *reinterpret_cast<float4*>(o_s + (warp * NH + h) * Dv + j * 128 + lane * 4) =
            make_float4(f * acc[h][4 * j], f * acc[h][4 * j + 1], f * acc[h][4 * j + 2], f * acc[h][4 * j + 3]);
  }
  __syncthreads();
  // ... goes to CTA 0 of the cluster, which adds the CTAs'
  if (ncta > 1) asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
  for (int i = threadIdx.x; i < nh * Dv; i += DL_THREADS) {
    float o = 0.f;
#pragma unroll
    for (int w = 0; w < DL_WARPS; ++w) o += o_s[w * NH * Dv + i];
    if (ncta > 1) st_cluster(x_s + rank * NH * Dv + i, 0, o);
    else x_s[i] = o;
  }
  if (warp < nh) {
    const int h = warp;
    const float ml = lane < DL_WARPS ? m_s[lane][h] : -CUDART_INF_F;
    float m = -CUDART_INF_F;
#pragma unroll
    for (int k = 0; k < NH; ++k) m = k == h ? mc[k] : m;
    float l = ml == -CUDART_INF_F ? 0.f : expf(ml - m) * l_s[lane][h];
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
    if (lane == 0) {
      if (ncta > 1) {
        st_cluster(&xm[rank][h], 0, m);
        st_cluster(&xl[rank][h], 0, l);
      } else {
        xm[0][h] = m;
        xl[0][h] = l;
      }
    }
  }
  if (ncta > 1) cluster_barrier();
  else __syncthreads();
  if (rank != 0) return;
  float* out = p.out + static_cast<int64_t>(g * p.groups + h0) * Dv;
  for (int i = threadIdx.x; i < nh * Dv; i += DL_THREADS) {
    const int h = i / Dv;
    float m = -CUDART_INF_F;
    for (int r = 0; r < ncta; ++r) m = fmaxf(m, xm[r][h]);
    float l = 0.f, o = 0.f;
#pragma unroll 4
    for (int r = 0; r < ncta; ++r) {
      const float f = xm[r][h] == -CUDART_INF_F ? 0.f : expf(xm[r][h] - m);
      l = fmaf(f, xl[r][h], l);
      o = fmaf(f, x_s[r * NH * Dv + i], o);
    }
    out[i] = o / l;
  }
}

// Launch with an optional cluster size, dependent on the kernel before it inside an overlap scope.
template <typename... KArgs, typename... Args>
static cudaError_t launch_cluster(void (*kernel)(KArgs...), int grid, int cluster, size_t smem, cudaStream_t st,
                                  Args&&... args) {
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = dim3(grid);
  cfg.blockDim = dim3(DL_THREADS);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = cluster;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = overlap_scope() ? 2 : 1;
  return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}

template <typename T, int NH>
static int decode_attention_t(const DecodeAttn& a, cudaStream_t st) {
  constexpr int KW = DA_KW<T>;
  const int units = a.kv_heads * ((a.groups + NH - 1) / NH);
  int ncta = 1;
  while (ncta < DA_MAX_CLUSTER && static_cast<int64_t>(ncta) * DL_WARPS * 4 < a.max_keys && units * ncta * 2 <= sm_count())
    ncta *= 2;
  const int64_t per_warp = (a.max_keys - 1) / (ncta * DL_WARPS) + 1;
  const int step = DL_WARPS * KW * (a.dim + a.vdim) * static_cast<int>(sizeof(T));
  // (the new key and value pass through the warps' output area on their way)
  const int outs = DL_WARPS * NH * a.vdim > a.dim + a.vdim ? DL_WARPS * NH * a.vdim : a.dim + a.vdim;
  const int rest = (NH * a.dim + outs + ncta * NH * a.vdim) * 4;
  const int nbuf = (per_warp > KW && 2 * step + rest <= 170 * 1024) ? 2 : 1;
  const int smem = nbuf * step + rest;
  auto* fn = a.vdim <= 128 ? decode_attn_kernel<T, NH, 1> : decode_attn_kernel<T, NH, 2>;
  const int s = dl_smem_check(reinterpret_cast<const void*>(fn), smem, "attention");
  if (s != YTC_OK) return s;
  YTC_CUDA(launch_cluster(fn, units * ncta, ncta, smem, st, a, ncta, nbuf));
  count_launch();
  YTC_CUDA(cudaGetLastError());
  return YTC_OK;
}

int decode_attention(const DecodeAttn& a, cudaStream_t st) {
  YTC_REQUIRE(a.dim > 0 && a.dim % 8 == 0 && a.vdim > 0 && a.vdim % 8 == 0 && a.vdim <= 256 && a.max_keys > 0 && a.ring > 0,
              "decode step: head dims must be multiples of 8, the value dim at most 256");
  if (a.dtype == YTC_BF16)
    return a.groups == 1 ? decode_attention_t<uint16_t, 1>(a, st)
                         : a.groups == 2 ? decode_attention_t<uint16_t, 2>(a, st) : decode_attention_t<uint16_t, 4>(a, st);
  return a.groups == 1 ? decode_attention_t<float, 1>(a, st)
                       : a.groups == 2 ? decode_attention_t<float, 2>(a, st) : decode_attention_t<float, 4>(a, st);
}

// ------------------------------------------------------------------ router
// One cluster: every CTA computes a share of the logits, CTA 0 collects them and routes.
constexpr int DR_CLUSTER = 8;

// The rule of warp_route (lm_ops.cuh) by a whole CTA: every route counts the routes in front of it, so that there is no
// chain of one selection after the other. s: logits, overwritten by the scores; c, g: scratch of n and `count` floats.
__device__ __forceinline__ float block_max(float v, float* red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float m = red[0];
#pragma unroll
  for (int i = 1; i < DL_WARPS; ++i) m = fmaxf(m, red[i]);
  return m;
}
__device__ __forceinline__ bool comes_before(float a, int i, float b, int j) { return a > b || (a == b && i < j); }
__device__ __forceinline__ void block_route(float* s, float* c, float* g, float* red, const float* correction,
                                            const RouterSpec& r, int* choice, float* weight) {
  const int n = r.experts + r.identity;
  if (!correction)
    for (int i = threadIdx.x; i < n; i += DL_THREADS) c[i] = s[i];
  if (r.score == ROUTE_SIGMOID) {
    for (int i = threadIdx.x; i < n; i += DL_THREADS) {
      const float p = lm_sigmoid(s[i]);
      s[i] = p;
      if (correction) c[i] = p + correction[i];
    }
  } else {
    float m = -INFINITY;
    for (int i = threadIdx.x; i < n; i += DL_THREADS) m = fmaxf(m, s[i]);
    m = block_max(m, red);
    float sum = 0.f;
    for (int i = threadIdx.x; i < n; i += DL_THREADS) {
      const float e = expf(s[i] - m);
      s[i] = e;
      sum += e;
    }
    sum = dl_block_sum(sum, red + DL_WARPS);
    for (int i = threadIdx.x; i < n; i += DL_THREADS) {
      const float p = s[i] / sum;
      s[i] = p;
      if (correction) c[i] = p + correction[i];
    }
  }
  if (threadIdx.x < r.top) {  // (places that no route takes)
    choice[threadIdx.x] = -1;
    weight[threadIdx.x] = 0.f;
  }
  __syncthreads();
  if (r.keep < r.count) {
    const int per = n / r.count;
    for (int k = threadIdx.x; k < r.count; k += DL_THREADS) {
      float b = -INFINITY;
      for (int i = 0; i < per; ++i) b = fmaxf(b, c[k * per + i]);
      g[k] = b;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < n; i += DL_THREADS) {
      const int mine = i / per;
      int before = 0;
      for (int k = 0; k < r.count; ++k) before += comes_before(g[k], k, g[mine], mine) ? 1 : 0;
      if (before >= r.keep) c[i] = -INFINITY;
    }
    __syncthreads();
  }
  for (int i = threadIdx.x; i < n; i += DL_THREADS) {
    const float mine = c[i];
    if (mine == -INFINITY) continue;
    int before = 0;
#pragma unroll 4
    for (int k = 0; k < n; ++k) before += comes_before(c[k], k, mine, i) ? 1 : 0;
    if (before < r.top) {
      choice[before] = i;
      weight[before] = s[i];
    }
  }
}

__global__ void __launch_bounds__(DL_THREADS, 2) decode_route_kernel(const DecodeRoute p, int ks, int padded) {
  extern __shared__ __align__(16) uint8_t dr_smem[];  // weight rings, input, part[], scores[n], choice scores[n], groups
  __shared__ float red[2 * DL_WARPS];
  const int n = p.r.experts + p.r.identity, pairs = (n + 1) / 2;
  const InputSmem in = input_smem(p.in.kind, reinterpret_cast<float*>(dr_smem + DL_WARPS * DL_RING), p.k, padded);
  float* part = in.h + input_floats(p.in.kind, p.k, padded);
  float* s = part + ((pairs + DR_CLUSTER - 1) / DR_CLUSTER) * 2 * ks;
  float* c = s + n;
  float* g = c + n;
  const int lane = threadIdx.x & 31;
  const int rank = blockIdx.x;
  int begin, end;
  my_pairs(pairs, begin, end);
  auto addr = [&](int pair, int piece, const uint16_t*& p0, const uint16_t*& p1, bool& ok0, bool& ok1) {
    const int col = piece * DL_PIECE + lane * 8;
    ok0 = col < p.k;
    ok1 = ok0 && 2 * pair + 1 < n;
    p0 = p.w + static_cast<int64_t>(2 * pair) * p.k + (ok0 ? col : 0);
    p1 = ok1 ? p0 + p.k : p0;
  };
  RowPairs<decltype(addr)> rp(addr, dr_smem, begin, end, (p.k + DL_PIECE - 1) / DL_PIECE, ks);
  prefetch_input(p.in, p.k, in);
  rp.start();
  float* corr = g + p.r.count;
  if (rank == 0)
    for (int i = threadIdx.x; i < n; i += DL_THREADS) corr[i] = p.correction ? p.correction[i] : 0.f;
  asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");  // (this CTA has started)
  dependent_wait();
  dependent_trigger();
  stage_input<DL_DEPTH - 1>(p.in, p.k, padded, in, red, rank == 0, p.h);
  rp.run(in.h, part);
  __syncthreads();
  asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
  for (int i = threadIdx.x; i < (end - begin) * 2; i += DL_THREADS)
    if (begin * 2 + i < n) st_cluster(s + begin * 2 + i, 0, sum_sub(part, i, ks));
  cluster_barrier();
  if (rank == 0) block_route(s, c, g, red, p.correction ? corr : nullptr, p.r, p.choice, p.weight);
}

int decode_route(const DecodeRoute& a, cudaStream_t st) {
  int s = check_input(a.in, a.k);
  if (s != YTC_OK) return s;
  const int n = a.r.experts + a.r.identity, pairs = (n + 1) / 2, per = (pairs + DR_CLUSTER - 1) / DR_CLUSTER;
  const int pieces = (a.k + DL_PIECE - 1) / DL_PIECE, padded = pieces * DL_PIECE;
  const int ks = pick_ks(per, pieces);
  const int smem = DL_WARPS * DL_RING +
                   (input_floats(a.in.kind, a.k, padded) + per * 2 * ks + 3 * n + a.r.count) * static_cast<int>(sizeof(float));
  YTC_REQUIRE(a.in.kind == DECODE_EMBED || a.in.kind == DECODE_RESIDUAL, "decode step: the router's input is a normed residual row");
  if ((s = dl_smem_check(reinterpret_cast<const void*>(decode_route_kernel), smem, "the router")) != YTC_OK) return s;
  YTC_CUDA(launch_cluster(decode_route_kernel, DR_CLUSTER, DR_CLUSTER, smem, st, a, ks, padded));
  count_launch();
  YTC_CUDA(cudaGetLastError());
  return YTC_OK;
}

// ------------------------------------------------------------------ experts
// The chosen experts (not the identity experts) of the token, compacted: expert[i], weight[i], slot[i] (its choice).
struct Chosen {
  int n;
  int expert[LM_MAX_TOP], slot[LM_MAX_TOP];
  float weight[LM_MAX_TOP];
  float identity;  // sum of the identity experts' weights
};
__device__ __forceinline__ void read_choice(const DecodeExperts& p, Chosen* c) {
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x;
    const int e = lane < p.r.top ? p.choice[lane] : -1;
    const float w = lane < p.r.top ? p.weight[lane] : 0.f;
    const bool real = e >= 0 && e < p.r.experts;
    const uint32_t mask = __ballot_sync(0xffffffffu, real);
    if (real) {
      const int i = __popc(mask & ((1u << lane) - 1u));
      c->expert[i] = e;
      c->slot[i] = lane;
      c->weight[i] = w;
    }
    float id = e >= p.r.experts ? w : 0.f;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) id += __shfl_xor_sync(0xffffffffu, id, o);
    if (lane == 0) {
      c->n = __popc(mask);
      c->identity = id;
    }
  }
  __syncthreads();
}

// mid[slot][j] = gated(gate_j . h, up_j . h): a row pair is (gate_j, up_j) of one chosen expert, the shared expert's pairs
// come first
__global__ void __launch_bounds__(DL_THREADS, 2) decode_gate_up_kernel(const DecodeExperts p, int ks, int padded) {
  extern __shared__ __align__(16) uint8_t dg_smem[];  // weight rings, input, part[]
  __shared__ Chosen ch;
  float* xs = reinterpret_cast<float*>(dg_smem + DL_WARPS * DL_RING);
  float* part = xs + padded;
  dependent_wait();
  dependent_trigger();
  read_choice(p, &ch);
  int begin, end;
  my_pairs(p.shared_ff + ch.n * p.ff, begin, end);
  const int lane8 = (threadIdx.x & 31) * 8;
  auto addr = [&](int pair, int piece, const uint16_t*& p0, const uint16_t*& p1, bool& ok0, bool& ok1) {
    const int col = piece * DL_PIECE + lane8;
    ok0 = ok1 = col < p.k;
    if (pair < p.shared_ff) {
      p0 = p.shared_gate_up + static_cast<int64_t>(2 * pair) * p.k + (ok0 ? col : 0);
    } else {
      const int q = pair - p.shared_ff, i = q / p.ff, j = q - i * p.ff;
      p0 = p.gate_up + (static_cast<int64_t>(ch.expert[i]) * 2 * p.ff + 2 * j) * p.k + (ok0 ? col : 0);
    }
    p1 = p0 + p.k;
  };
  RowPairs<decltype(addr)> rp(addr, dg_smem, begin, end, (p.k + DL_PIECE - 1) / DL_PIECE, ks);
  rp.start();
  for (int c = threadIdx.x * 4; c < padded; c += DL_THREADS * 4)
    *reinterpret_cast<float4*>(xs + staged_at(c)) =
        c < p.k ? *reinterpret_cast<const float4*>(p.h + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  __syncthreads();
  rp.run(xs, part);
  __syncthreads();
  for (int i = threadIdx.x; i < end - begin; i += DL_THREADS) {
    const int pair = begin + i;
    const float g = sum_sub(part, 2 * i, ks), u = sum_sub(part, 2 * i + 1, ks);
    if (pair < p.shared_ff) {
      p.mid[static_cast<int64_t>(p.r.top) * p.ff + pair] = lm_gated(p.shared_act, g, u);
    } else {
      const int q = pair - p.shared_ff, e = q / p.ff, j = q - e * p.ff;
      const float w = p.scale_input ? ch.weight[e] : 1.f;  // (both products are linear in the expert's input)
      p.mid[static_cast<int64_t>(ch.slot[e]) * p.ff + j] = lm_gated(p.act, w * g, w * u);
    }
  }
}

// out[n] = sum over the chosen experts of weight * (down_n . mid) + (identity weights) * h[n] + (shared down_n . mid): the
// experts' vectors, already multiplied by their weights, stand one after the other in shared memory, the shared one first
__global__ void __launch_bounds__(DL_THREADS, 2) decode_down_kernel(const DecodeExperts p, int ks, int ff_padded,
                                                                    int shared_padded) {
  extern __shared__ __align__(16) uint8_t dd_smem[];  // weight rings, inputs [shared_padded], [top][ff_padded], part[]
  __shared__ Chosen ch;
  float* xs = reinterpret_cast<float*>(dd_smem + DL_WARPS * DL_RING);
  float* part = xs + shared_padded + p.r.top * ff_padded;
  // (the choice was made two kernels ago: the kernel before this one has already waited for it)
  read_choice(p, &ch);
  int begin, end;
  my_pairs(p.k / 2, begin, end);
  const int lane8 = (threadIdx.x & 31) * 8;
  const int per_expert = ff_padded / DL_PIECE, shared_pieces = shared_padded / DL_PIECE;
  auto addr = [&](int pair, int piece, const uint16_t*& p0, const uint16_t*& p1, bool& ok0, bool& ok1) {
    if (piece < shared_pieces) {
      const int col = piece * DL_PIECE + lane8;
      ok0 = ok1 = col < p.shared_ff;
      p0 = p.shared_down + static_cast<int64_t>(2 * pair) * p.shared_ff + (ok0 ? col : 0);
      p1 = p0 + p.shared_ff;
      return;
    }
    const int q = piece - shared_pieces, i = q / per_expert, col = (q - i * per_expert) * DL_PIECE + lane8;
    ok0 = ok1 = col < p.ff;
    p0 = p.down + (static_cast<int64_t>(ch.expert[i]) * p.k + 2 * pair) * p.ff + (ok0 ? col : 0);
    p1 = p0 + p.ff;
  };
  const int pieces = shared_pieces + ch.n * per_expert;
  const int ks_here = pieces < ks ? 1 : ks;
  RowPairs<decltype(addr)> rp(addr, dd_smem, begin, pieces > 0 ? end : begin, pieces, ks_here);
  rp.start();
  dependent_wait();
  dependent_trigger();
  for (int c = threadIdx.x * 4; c < shared_padded; c += DL_THREADS * 4)
    *reinterpret_cast<float4*>(xs + staged_at(c)) =
        c < p.shared_ff ? *reinterpret_cast<const float4*>(p.mid + static_cast<int64_t>(p.r.top) * p.ff + c)
                        : make_float4(0.f, 0.f, 0.f, 0.f);
  const int per4 = ff_padded / 4;
  for (int v = threadIdx.x; v < ch.n * per4; v += DL_THREADS) {
    const int i = v / per4, c = (v - i * per4) * 4;
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < p.ff) a = *reinterpret_cast<const float4*>(p.mid + static_cast<int64_t>(ch.slot[i]) * p.ff + c);
    const float w = p.scale_input ? 1.f : ch.weight[i];
    *reinterpret_cast<float4*>(xs + shared_padded + i * ff_padded + staged_at(c)) =
        make_float4(w * a.x, w * a.y, w * a.z, w * a.w);
  }
  __syncthreads();
  rp.run(xs, part);
  __syncthreads();
  for (int i = threadIdx.x; i < (end - begin) * 2; i += DL_THREADS) {
    const int row = begin * 2 + i;
    p.out[row] = (pieces > 0 ? sum_sub(part, i, ks_here) : 0.f) + ch.identity * p.h[row];
  }
}

int decode_experts(const DecodeExperts& a, cudaStream_t st) {
  YTC_REQUIRE(a.k % 8 == 0 && a.ff % 8 == 0 && a.shared_ff % 8 == 0 && a.r.top <= LM_MAX_TOP, "decode step: bad expert size");
  int s;
  {
    const int pieces = (a.k + DL_PIECE - 1) / DL_PIECE, padded = pieces * DL_PIECE, pairs = a.shared_ff + a.r.top * a.ff;
    const int grid = pairs < sm_count() ? pairs : sm_count();
    const int per = (pairs + grid - 1) / grid, ks = pick_ks(per, pieces);
    const int smem = DL_WARPS * DL_RING + (padded + per * 2 * ks) * static_cast<int>(sizeof(float));
    if ((s = dl_smem_check(reinterpret_cast<const void*>(decode_gate_up_kernel), smem, "an expert's input")) != YTC_OK) return s;
    YTC_CUDA(launch_overlapped(decode_gate_up_kernel, dim3(grid), dim3(DL_THREADS), smem, st, a, ks, padded));
    count_launch();
    YTC_CUDA(cudaGetLastError());
  }
  const int per_expert = (a.ff + DL_PIECE - 1) / DL_PIECE, ff_padded = per_expert * DL_PIECE, pairs = a.k / 2;
  const int shared_padded = (a.shared_ff + DL_PIECE - 1) / DL_PIECE * DL_PIECE;
  const int grid = pairs < sm_count() ? pairs : sm_count();
  const int per = (pairs + grid - 1) / grid, ks = pick_ks(per, a.r.top * per_expert + shared_padded / DL_PIECE);
  const int smem = DL_WARPS * DL_RING +
                   (shared_padded + a.r.top * ff_padded + per * 2 * ks) * static_cast<int>(sizeof(float));
  if ((s = dl_smem_check(reinterpret_cast<const void*>(decode_down_kernel), smem, "the experts' activations")) != YTC_OK) return s;
  YTC_CUDA(launch_overlapped(decode_down_kernel, dim3(grid), dim3(DL_THREADS), smem, st, a, ks, ff_padded, shared_padded));
  count_launch();
  YTC_CUDA(cudaGetLastError());
  return YTC_OK;
}

}  // namespace ytk
