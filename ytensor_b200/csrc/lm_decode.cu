// One new token of a windowed language model: the kernels of a decode step.
//
// A step is a chain of short kernels (projection with the norms before it, attention, projection, ...) queued as
// programmatic dependent launches inside a CUDA graph. Every kernel requests the weights (or the old keys and values) it
// will multiply by BEFORE it waits for the kernel in front of it, so that the weight stream does not stop at kernel
// boundaries: two kernels of the chain are resident at a time (256 threads, at most 128 registers). Activations are
// fp32 vectors of a few KB; every CTA stages the whole vector in shared memory and recomputes the norms from it, which
// costs less than one more hand-over.
#include <math_constants.h>

#include "lm_ops.cuh"

namespace ytk {

constexpr int DL_THREADS = 256, DL_WARPS = DL_THREADS / 32;
constexpr int DL_UN = 4;          // row-pair pieces per batch of loads; two batches are in flight
constexpr int DL_PIECE = 256;     // columns a warp covers with one 16-byte load per lane

__device__ __forceinline__ uint4 ld_weights(const uint16_t* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];"
               : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w)
               : "l"(p));
  return v;
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

// Stages the input vector of `k` floats into xs[0 .. padded), zero beyond k. `writer`: this CTA stores the new residual
// row (and the normed vector, when h_out is given).
__device__ __forceinline__ void stage_input(const DecodeInput& in, int k, int padded, float* xs, float* red, bool writer,
                                            float* h_out) {
  for (int c = k + threadIdx.x; c < padded; c += DL_THREADS) xs[c] = 0.f;
  if (in.kind == 2) {
    for (int c = threadIdx.x * 4; c < k; c += DL_THREADS * 4)
      *reinterpret_cast<float4*>(xs + c) = *reinterpret_cast<const float4*>(in.plain + c);
    __syncthreads();
    return;
  }
  if (in.kind == 0) {
    int id = *in.id;
    id = id < 0 ? 0 : (id >= in.vocab ? in.vocab - 1 : id);
    const uint16_t* row = in.embed + static_cast<int64_t>(id) * k;
    for (int c = threadIdx.x; c < k; c += DL_THREADS) {
      const float v = bf16_bits_to_f32(row[c]);
      xs[c] = v;
      if (writer) in.x_out[c] = v;
    }
  } else {
    float ss = 0.f;
    for (int c = threadIdx.x * 4; c < k; c += DL_THREADS * 4) {
      const float4 y = *reinterpret_cast<const float4*>(in.y + c);
      *reinterpret_cast<float4*>(xs + c) = y;  // (read back by this thread only)
      ss = fmaf(y.x, y.x, ss); ss = fmaf(y.y, y.y, ss); ss = fmaf(y.z, y.z, ss); ss = fmaf(y.w, y.w, ss);
    }
    const float inv = 1.0f / sqrtf(dl_block_sum(ss, red) / in.width + in.eps);
    for (int c = threadIdx.x * 4; c < k; c += DL_THREADS * 4) {
      const float4 y = *reinterpret_cast<const float4*>(xs + c), g = *reinterpret_cast<const float4*>(in.w_post + c);
      float4 x = *reinterpret_cast<const float4*>(in.x_in + c);
      x.x += y.x * inv * g.x; x.y += y.y * inv * g.y; x.z += y.z * inv * g.z; x.w += y.w * inv * g.w;
      *reinterpret_cast<float4*>(xs + c) = x;
      if (writer) *reinterpret_cast<float4*>(in.x_out + c) = x;
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = threadIdx.x * 4; c < k; c += DL_THREADS * 4) {
    const float4 x = *reinterpret_cast<const float4*>(xs + c);
    ss = fmaf(x.x, x.x, ss); ss = fmaf(x.y, x.y, ss); ss = fmaf(x.z, x.z, ss); ss = fmaf(x.w, x.w, ss);
  }
  const float inv = 1.0f / sqrtf(dl_block_sum(ss, red + DL_WARPS) / in.width + in.eps);
  for (int c = threadIdx.x * 4; c < k; c += DL_THREADS * 4) {
    const float4 g = *reinterpret_cast<const float4*>(in.w_pre + c);
    float4 x = *reinterpret_cast<const float4*>(xs + c);
    x.x *= inv * g.x; x.y *= inv * g.y; x.z *= inv * g.z; x.w *= inv * g.w;
    *reinterpret_cast<float4*>(xs + c) = x;
    if (writer && h_out) *reinterpret_cast<float4*>(h_out + c) = x;
  }
  __syncthreads();
}

// The product loop. A CTA owns output row pairs [begin, end); KS warps share a pair and split its pieces of 256
// columns. addr(pair, piece, r): the lane's 16 bytes of weight row 2 pair + r (null beyond the row's end). Partial sums
// go to part[(pair - begin) * 2 + r][sub].
template <typename Addr>
struct RowPairs {
  Addr addr;
  int end, pieces, ks, sub, slots;
  int lp, lpc;               // loader's cursor
  int cp, cpc;               // consumer's cursor
  float a0 = 0.f, a1 = 0.f;
  __device__ RowPairs(Addr f, int begin, int end_, int pieces_, int ks_) : addr(f), end(end_), pieces(pieces_), ks(ks_) {
    const int warp = threadIdx.x >> 5;
    sub = warp % ks;
    slots = DL_WARPS / ks;
    lp = cp = begin + warp / ks;
    lpc = cpc = sub;
    if (sub >= pieces) lp = cp = end;  // (ks never exceeds the pieces; kept for safety)
  }
  __device__ __forceinline__ bool more() const { return cp < end; }
  __device__ __forceinline__ void load(uint4 (&buf)[DL_UN][2]) {
#pragma unroll
    for (int u = 0; u < DL_UN; ++u) {
      buf[u][0] = buf[u][1] = make_uint4(0u, 0u, 0u, 0u);
      if (lp >= end) continue;
      const uint16_t* p0 = addr(lp, lpc, 0);
      const uint16_t* p1 = addr(lp, lpc, 1);
      if (p0) buf[u][0] = ld_weights(p0);
      if (p1) buf[u][1] = ld_weights(p1);
      lpc += ks;
      if (lpc >= pieces) {
        lpc = sub;
        lp += slots;
      }
    }
  }
  // xs: the staged vector, piece p at xs + 256 p
  __device__ __forceinline__ void consume(const uint4 (&buf)[DL_UN][2], const float* xs, float* part, int begin) {
    const int lane = threadIdx.x & 31;
#pragma unroll
    for (int u = 0; u < DL_UN; ++u) {
      if (cp >= end) return;
      float x[8], w[8];
      Vec8<float>::load(xs + cpc * DL_PIECE + lane * 8, x);
      Vec8<uint16_t>::unpack(buf[u][0], w);
#pragma unroll
      for (int e = 0; e < 8; ++e) a0 = fmaf(x[e], w[e], a0);
      Vec8<uint16_t>::unpack(buf[u][1], w);
#pragma unroll
      for (int e = 0; e < 8; ++e) a1 = fmaf(x[e], w[e], a1);
      cpc += ks;
      if (cpc >= pieces) {
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
          a0 += __shfl_xor_sync(0xffffffffu, a0, o);
          a1 += __shfl_xor_sync(0xffffffffu, a1, o);
        }
        if (lane == 0) {
          part[((cp - begin) * 2) * ks + sub] = a0;
          part[((cp - begin) * 2 + 1) * ks + sub] = a1;
        }
        a0 = a1 = 0.f;
        cpc = sub;
        cp += slots;
      }
    }
  }
};

__device__ __forceinline__ float sum_sub(const float* part, int row, int ks) {
  float s = 0.f;
  for (int i = 0; i < ks; ++i) s += part[row * ks + i];
  return s;
}

// Warps that share a row pair: the count with the fewest rounds of pieces per warp.
static int pick_ks(int pairs_per_cta, int pieces) {
  int best = 1;
  double best_cost = 1e30;
  for (int ks = 1; ks <= DL_WARPS && ks <= pieces; ks *= 2) {
    const int slots = DL_WARPS / ks;
    const double rounds = (pairs_per_cta + slots - 1) / slots;
    const double cost = rounds * ((pieces + ks - 1) / ks);
    if (cost < best_cost * 0.95) {
      best_cost = cost;
      best = ks;
    }
  }
  return best;
}

// ------------------------------------------------------------------ linear
__global__ void __launch_bounds__(DL_THREADS, 2) decode_linear_kernel(const DecodeLinear p, int ks, int padded) {
  extern __shared__ float dl_smem[];  // xs[padded], part[]
  __shared__ float red[2 * DL_WARPS];
  float* xs = dl_smem;
  float* part = dl_smem + padded;
  const int pairs = (p.n + 1) / 2;
  const int begin = static_cast<int>(static_cast<int64_t>(pairs) * blockIdx.x / gridDim.x);
  const int end = static_cast<int>(static_cast<int64_t>(pairs) * (blockIdx.x + 1) / gridDim.x);
  const int lane8 = (threadIdx.x & 31) * 8;
  auto addr = [&](int pair, int piece, int r) -> const uint16_t* {
    const int row = 2 * pair + r, col = piece * DL_PIECE + lane8;
    return (row < p.n && col < p.k) ? p.w + static_cast<int64_t>(row) * p.k + col : nullptr;
  };
  RowPairs<decltype(addr)> rp(addr, begin, end, (p.k + DL_PIECE - 1) / DL_PIECE, ks);
  uint4 b0[DL_UN][2], b1[DL_UN][2];
  rp.load(b0);
  rp.load(b1);
  dependent_wait();
  dependent_trigger();
  stage_input(p.in, p.k, padded, xs, red, blockIdx.x == 0, nullptr);
  while (rp.more()) {
    rp.consume(b0, xs, part, begin);
    rp.load(b0);
    rp.consume(b1, xs, part, begin);
    rp.load(b1);
  }
  __syncthreads();
  for (int i = threadIdx.x; i < (end - begin) * 2; i += DL_THREADS) {
    const int row = begin * 2 + i;
    if (row >= p.n) continue;
    const float v = sum_sub(part, i, ks);
    p.out[row] = p.epi == EPI_GELU_ERF ? lm_gelu_erf(v) : v;
  }
  if (p.advance && blockIdx.x == 0 && threadIdx.x == 0) *p.advance += 1;
}

static int check_input(const DecodeInput& in, int k) {
  YTC_REQUIRE(k > 0 && k % 8 == 0 && (in.kind == 2 || in.width <= k), "decode step: bad vector length %d", k);
  return YTC_OK;
}

int decode_linear(const DecodeLinear& a, cudaStream_t st) {
  int s = check_input(a.in, a.k);
  if (s != YTC_OK) return s;
  const int pieces = (a.k + DL_PIECE - 1) / DL_PIECE, padded = pieces * DL_PIECE, pairs = (a.n + 1) / 2;
  const int grid = pairs < sm_count() ? pairs : sm_count();
  const int per = (pairs + grid - 1) / grid;
  const int ks = pick_ks(per, pieces);
  const int smem = (padded + per * 2 * ks) * static_cast<int>(sizeof(float));
  if (smem > 200 * 1024) {
    set_last_error("decode step: a projection of %d x %d does not fit shared memory", a.n, a.k);
    return YTC_UNSUPPORTED;
  }
  if (smem > 48 * 1024 && (s = ensure_dynamic_smem(reinterpret_cast<const void*>(decode_linear_kernel), smem)) != YTC_OK)
    return s;
  YTC_CUDA(launch_overlapped(decode_linear_kernel, dim3(grid), dim3(DL_THREADS), smem, st, a, ks, padded));
  count_launch();
  YTC_CUDA(cudaGetLastError());
  return YTC_OK;
}

// ------------------------------------------------------------------ attention
// One cluster of CTAs per K/V head; the keys of the window are split over its CTAs, each handles all query heads of the
// group. Per chunk of keys: keys and values in shared memory (the old ones requested before the wait for the projection),
// eight lanes per key for the scores of all heads, then the value dim across threads. The CTAs' (max, sum, O) meet
// through distributed shared memory.
constexpr int DA_MAX_CLUSTER = 8;
constexpr int DA_GB = 4;  // query heads per pass over the values

__device__ __forceinline__ float ld_cluster(const float* p, uint32_t rank) {
  uint32_t a = static_cast<uint32_t>(__cvta_generic_to_shared(p)), r;
  float v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(a), "r"(rank));
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(r) : "memory");
  return v;
}
__device__ __forceinline__ void cluster_barrier() {
  asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
  asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))),
               "l"(src)
               : "memory");
}

template <typename T>
__global__ void __launch_bounds__(DL_THREADS, 2) decode_attn_kernel(const DecodeAttn p, int chunk, int ncta) {
  // q[G][dim], o[G][vdim], score[G][chunk], m[G], l[G], red[8][DA_GB][vdim] (floats), then K[chunk][dim + 16 B],
  // V[chunk][vdim]
  extern __shared__ __align__(16) float da_smem[];
  const int G = p.groups, D = p.dim, Dv = p.vdim;
  float* q_s = da_smem;
  float* o_s = q_s + G * D;
  float* sc = o_s + G * Dv;
  float* m_s = sc + G * chunk;
  float* l_s = m_s + G;
  float* red = l_s + G;
  red = reinterpret_cast<float*>((reinterpret_cast<uintptr_t>(red) + 15) & ~static_cast<uintptr_t>(15));
  constexpr int PADE = 16 / sizeof(T);
  const int kld = D + PADE;
  T* k_s = reinterpret_cast<T*>(red + DL_WARPS * DA_GB * Dv);
  T* v_s = k_s + chunk * kld;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = blockIdx.x / ncta, rank = blockIdx.x - g * ncta;

  // (the position word was written before this step's first kernel started)
  const int pos = *p.pos;
  const int seen = (p.window > 0 && pos + 1 > p.window) ? p.window : pos + 1;
  const int old_first = pos + 1 - seen, old_n = seen - 1;  // positions old_first .. pos - 1, then the new one
  const int per = (old_n + ncta - 1) / ncta;
  int k0 = rank * per;
  int k1 = k0 + per < old_n ? k0 + per : old_n;
  if (k0 > k1) k0 = k1;
  const int mine = k1 - k0 + (rank == 0 ? 1 : 0);  // CTA 0 also takes the new key, after its old ones
  const T* kr = static_cast<const T*>(p.k) + static_cast<int64_t>(g) * p.ring * D;
  const T* vr = static_cast<const T*>(p.v) + static_cast<int64_t>(g) * p.ring * Dv;
  constexpr int VE = 16 / sizeof(T);  // elements per 16 bytes
  auto fetch = [&](int c0) {  // requests old keys c0 .. of this CTA
    const int n_old = (k1 - k0) - c0 < chunk ? (k1 - k0) - c0 : chunk;
    const int kp = D / VE, vp = Dv / VE;
    for (int i = threadIdx.x; i < n_old * (kp + vp); i += DL_THREADS) {
      const int key = i / (kp + vp), c = i - key * (kp + vp);
      const int64_t row = (old_first + k0 + c0 + key) % p.ring;
      if (c < kp) cp_async16(k_s + key * kld + c * VE, kr + row * D + c * VE);
      else cp_async16(v_s + key * Dv + (c - kp) * VE, vr + row * Dv + (c - kp) * VE);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0);
  dependent_wait();
  dependent_trigger();
  const int H = p.kv_heads * G;
  for (int i = threadIdx.x; i < G * D; i += DL_THREADS) q_s[i] = p.qkv[static_cast<int64_t>(g) * G * D + i];
  for (int i = threadIdx.x; i < G * Dv; i += DL_THREADS) o_s[i] = 0.f;
  if (threadIdx.x < G) {
    m_s[threadIdx.x] = -CUDART_INF_F;
    l_s[threadIdx.x] = 0.f;
  }
  const float* k_new = p.qkv + static_cast<int64_t>(H) * D + static_cast<int64_t>(g) * D;
  const float* v_new = p.qkv + static_cast<int64_t>(H + p.kv_heads) * D + static_cast<int64_t>(g) * Dv;
  const float lam = p.mix == VMIX_MIX ? *p.lambda : 0.f;
  int npv = 1;  // lanes per value row (a power of two), 8 elements each
  while (npv * 8 < Dv) npv <<= 1;
  const int piece = threadIdx.x % npv, key_lane = threadIdx.x / npv, key_lanes = DL_THREADS / npv;

  for (int c0 = 0; c0 < mine; c0 += chunk) {
    const int n = mine - c0 < chunk ? mine - c0 : chunk;
    if (c0 > 0) {
      __syncthreads();  // everyone is done with the previous chunk
      fetch(c0);
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    if (rank == 0 && c0 + n == mine) {  // the new key and value: into the chunk and into the rings
      const int at = n - 1;
      const int64_t row = pos % p.ring;
      T* kw = static_cast<T*>(p.k) + (static_cast<int64_t>(g) * p.ring + row) * D;
      T* vw = static_cast<T*>(p.v) + (static_cast<int64_t>(g) * p.ring + row) * Dv;
      for (int i = threadIdx.x; i < (D + Dv) / 8; i += DL_THREADS) {
        float f[8];
        if (i < D / 8) {
          Vec8<float>::load(k_new + i * 8, f);
          Vec8<T>::store(kw + i * 8, f);
          Vec8<T>::store(k_s + at * kld + i * 8, f);
        } else {
          const int e = i * 8 - D;
          Vec8<float>::load(v_new + e, f);
          float* first = p.v_first + static_cast<int64_t>(g) * Dv + e;
          if (p.mix == VMIX_FIRST) Vec8<float>::store(first, f);
          if (p.mix == VMIX_MIX) {
            float v0[8];
            Vec8<float>::load(first, v0);
#pragma unroll
            for (int k = 0; k < 8; ++k) f[k] = (1.f - lam) * f[k] + lam * v0[k];
          }
          Vec8<T>::store(vw + e, f);
          Vec8<T>::store(v_s + at * Dv + e, f);
        }
      }
    }
    __syncthreads();
    // scores: eight lanes per key
    for (int key0 = warp * 4; key0 < n; key0 += DL_WARPS * 4) {
      const int key = key0 + (lane >> 3);
      const T* kv = k_s + (key < n ? key : 0) * kld;
      for (int h = 0; h < G; ++h) {
        float dot = 0.f;
        for (int c = (lane & 7) * 8; c < D; c += 64) {
          float a[8], b[8];
          Vec8<T>::load(kv + c, a);
          Vec8<float>::load(q_s + h * D + c, b);
#pragma unroll
          for (int e = 0; e < 8; ++e) dot = fmaf(a[e], b[e], dot);
        }
        dot += __shfl_xor_sync(0xffffffffu, dot, 1);
        dot += __shfl_xor_sync(0xffffffffu, dot, 2);
        dot += __shfl_xor_sync(0xffffffffu, dot, 4);
        if ((lane & 7) == 0 && key < n) {
          dot *= p.scale;
          sc[h * chunk + key] = p.softcap > 0.f ? p.softcap * tanhf(dot / p.softcap) : dot;
        }
      }
    }
    __syncthreads();
    for (int h = warp; h < G; h += DL_WARPS) {  // weights of a head: one warp
      float m = -CUDART_INF_F;
      for (int i = lane; i < n; i += 32) m = fmaxf(m, sc[h * chunk + i]);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
      const float m_old = m_s[h], m_new = fmaxf(m_old, m);
      const float alpha = m_old == -CUDART_INF_F ? 0.f : expf(m_old - m_new);
      float l = 0.f;
      for (int i = lane; i < n; i += 32) {
        const float w = expf(sc[h * chunk + i] - m_new);
        sc[h * chunk + i] = w;
        l += w;
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
      for (int i = lane; i < Dv; i += 32) o_s[h * Dv + i] *= alpha;
      __syncwarp();
      if (lane == 0) {
        m_s[h] = m_new;
        l_s[h] = l_s[h] * alpha + l;
      }
    }
    __syncthreads();
    for (int h0 = 0; h0 < G; h0 += DA_GB) {
      float acc[DA_GB][8] = {};
      if (piece * 8 < Dv)
        for (int key = key_lane; key < n; key += key_lanes) {
          float v[8];
          Vec8<T>::load(v_s + key * Dv + piece * 8, v);
#pragma unroll
          for (int hh = 0; hh < DA_GB; ++hh) {
            const float w = h0 + hh < G ? sc[(h0 + hh) * chunk + key] : 0.f;
#pragma unroll
            for (int e = 0; e < 8; ++e) acc[hh][e] = fmaf(w, v[e], acc[hh][e]);
          }
        }
      for (int o = npv; o < 32; o <<= 1)
#pragma unroll
        for (int hh = 0; hh < DA_GB; ++hh)
#pragma unroll
          for (int e = 0; e < 8; ++e) acc[hh][e] += __shfl_xor_sync(0xffffffffu, acc[hh][e], o);
      if (lane < npv && piece * 8 < Dv)
#pragma unroll
        for (int hh = 0; hh < DA_GB; ++hh) Vec8<float>::store(red + (warp * DA_GB + hh) * Dv + piece * 8, acc[hh]);
      __syncthreads();
      for (int i = threadIdx.x; i < DA_GB * Dv; i += DL_THREADS) {
        const int hh = i / Dv;
        if (h0 + hh >= G) break;
        float s = 0.f;
#pragma unroll
        for (int w = 0; w < DL_WARPS; ++w) s += red[w * DA_GB * Dv + i];
        o_s[h0 * Dv + i] += s;
      }
      __syncthreads();
    }
  }
  // the cluster's partial results: each CTA finishes a share of the outputs
  if (ncta > 1) cluster_barrier();
  else __syncthreads();
  for (int i = rank * DL_THREADS + threadIdx.x; i < G * Dv; i += ncta * DL_THREADS) {
    const int h = i / Dv;
    float m = -CUDART_INF_F;
    float ms[DA_MAX_CLUSTER];
#pragma unroll
    for (int r = 0; r < DA_MAX_CLUSTER; ++r) {
      ms[r] = r < ncta ? (ncta > 1 ? ld_cluster(m_s + h, r) : m_s[h]) : -CUDART_INF_F;
      m = fmaxf(m, ms[r]);
    }
    float l = 0.f, o = 0.f;
#pragma unroll
    for (int r = 0; r < DA_MAX_CLUSTER; ++r) {
      if (r >= ncta || ms[r] == -CUDART_INF_F) continue;
      const float f = expf(ms[r] - m);
      l += f * (ncta > 1 ? ld_cluster(l_s + h, r) : l_s[h]);
      o += f * (ncta > 1 ? ld_cluster(o_s + i, r) : o_s[i]);
    }
    p.out[static_cast<int64_t>(g) * G * Dv + i] = o / l;
  }
  if (ncta > 1) cluster_barrier();  // no CTA leaves while another may still read its shared memory
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

template <typename T>
static int decode_attention_t(const DecodeAttn& a, cudaStream_t st) {
  int ncta = 1;
  while (ncta < DA_MAX_CLUSTER && static_cast<int64_t>(ncta) * 32 < a.max_keys && a.kv_heads * ncta * 2 <= sm_count()) ncta *= 2;
  const int64_t mine = (a.max_keys + ncta - 1) / ncta + 1;
  auto bytes = [&](int chunk) {
    const size_t fl = static_cast<size_t>(a.groups) * (a.dim + a.vdim + chunk + 2) + DL_WARPS * DA_GB * a.vdim + 8;
    return fl * 4 + static_cast<size_t>(chunk) * (a.dim + 16 / sizeof(T) + a.vdim) * sizeof(T) + 32;
  };
  int chunk = static_cast<int>(mine < 256 ? (mine + 7) / 8 * 8 : 256);
  while (chunk > 8 && bytes(chunk) > 100 * 1024) chunk -= 8;  // two kernels of the chain share an SM
  if (bytes(chunk) > 220 * 1024) {
    set_last_error("decode step: %d query heads of %d + %d channels per K/V head do not fit shared memory", a.groups, a.dim,
                   a.vdim);
    return YTC_UNSUPPORTED;
  }
  const int smem = static_cast<int>(bytes(chunk));
  const int s = ensure_dynamic_smem(reinterpret_cast<const void*>(decode_attn_kernel<T>), smem);
  if (s != YTC_OK) return s;
  YTC_CUDA(launch_cluster(decode_attn_kernel<T>, a.kv_heads * ncta, ncta, smem, st, a, chunk, ncta));
  count_launch();
  YTC_CUDA(cudaGetLastError());
  return YTC_OK;
}

int decode_attention(const DecodeAttn& a, cudaStream_t st) {
  YTC_REQUIRE(a.dim > 0 && a.dim % 8 == 0 && a.vdim > 0 && a.vdim % 8 == 0 && a.vdim <= 256 && a.max_keys > 0 && a.ring > 0,
              "decode step: head dims must be multiples of 8, the value dim at most 256");
  return a.dtype == YTC_BF16 ? decode_attention_t<uint16_t>(a, st) : decode_attention_t<float>(a, st);
}

// ------------------------------------------------------------------ router
// One cluster: every CTA computes a share of the logits, CTA 0 collects them and routes.
constexpr int DR_CLUSTER = 8;
__global__ void __launch_bounds__(DL_THREADS, 2) decode_route_kernel(const DecodeRoute p, int padded) {
  extern __shared__ float dr_smem[];  // xs[padded], scores[n], choice scores[n]
  __shared__ float red[2 * DL_WARPS];
  const int n = p.r.experts + p.r.identity;
  float* xs = dr_smem;
  float* s = dr_smem + padded;
  float* c = s + n;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rank = blockIdx.x;
  dependent_wait();
  dependent_trigger();
  stage_input(p.in, p.k, padded, xs, red, rank == 0, p.h);
  for (int e = rank * DL_WARPS + warp; e < n; e += DR_CLUSTER * DL_WARPS) {
    const uint16_t* w = p.w + static_cast<int64_t>(e) * p.k;
    float acc = 0.f;
    for (int col = lane * 8; col < p.k; col += DL_PIECE) {
      float a[8], x[8];
      Vec8<uint16_t>::load(w + col, a);
      Vec8<float>::load(xs + col, x);
#pragma unroll
      for (int k = 0; k < 8; ++k) acc = fmaf(a[k], x[k], acc);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
    if (lane == 0) s[e] = acc;
  }
  cluster_barrier();
  if (rank == 0) {
    for (int e = threadIdx.x; e < n; e += DL_THREADS) {
      const uint32_t owner = (e / DL_WARPS) % DR_CLUSTER;
      if (owner != 0) s[e] = ld_cluster(s + e, owner);
    }
    __syncthreads();
    if (warp == 0) {
      int choice;
      float weight;
      warp_route(s, c, p.correction, p.r, lane, choice, weight);
      if (lane < p.r.top) {
        p.choice[lane] = choice;
        p.weight[lane] = weight;
      }
    }
  }
  cluster_barrier();
}

int decode_route(const DecodeRoute& a, cudaStream_t st) {
  int s = check_input(a.in, a.k);
  if (s != YTC_OK) return s;
  const int n = a.r.experts + a.r.identity;
  const int padded = (a.k + DL_PIECE - 1) / DL_PIECE * DL_PIECE;
  const int smem = (padded + 2 * n) * static_cast<int>(sizeof(float));
  if (smem > 48 * 1024 && (s = ensure_dynamic_smem(reinterpret_cast<const void*>(decode_route_kernel), smem)) != YTC_OK)
    return s;
  YTC_CUDA(launch_cluster(decode_route_kernel, DR_CLUSTER, DR_CLUSTER, smem, st, a, padded));
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
  if (threadIdx.x == 0) {
    int n = 0;
    float id = 0.f;
    for (int k = 0; k < p.r.top; ++k) {
      const int e = p.choice[k];
      const float w = p.weight[k];
      if (e >= p.r.experts) id += w;
      else if (e >= 0) {
        c->expert[n] = e;
        c->slot[n] = k;
        c->weight[n++] = w;
      }
    }
    c->n = n;
    c->identity = id;
  }
  __syncthreads();
}

// act[slot][j] = silu(gate_j . h) * (up_j . h): a row pair is (gate_j, up_j) of one chosen expert
__global__ void __launch_bounds__(DL_THREADS, 2) decode_gate_up_kernel(const DecodeExperts p, int ks, int padded) {
  extern __shared__ float dg_smem[];
  __shared__ Chosen ch;
  float* xs = dg_smem;
  float* part = dg_smem + padded;
  dependent_wait();
  dependent_trigger();
  read_choice(p, &ch);
  const int pairs = ch.n * p.ff;
  const int begin = static_cast<int>(static_cast<int64_t>(pairs) * blockIdx.x / gridDim.x);
  const int end = static_cast<int>(static_cast<int64_t>(pairs) * (blockIdx.x + 1) / gridDim.x);
  const int lane8 = (threadIdx.x & 31) * 8;
  auto addr = [&](int pair, int piece, int r) -> const uint16_t* {
    const int col = piece * DL_PIECE + lane8;
    if (col >= p.k) return nullptr;
    const int i = pair / p.ff, j = pair - i * p.ff;
    return p.gate_up + (static_cast<int64_t>(ch.expert[i]) * 2 * p.ff + 2 * j + r) * p.k + col;
  };
  RowPairs<decltype(addr)> rp(addr, begin, end, (p.k + DL_PIECE - 1) / DL_PIECE, ks);
  uint4 b0[DL_UN][2], b1[DL_UN][2];
  rp.load(b0);
  rp.load(b1);
  for (int c = threadIdx.x; c < padded; c += DL_THREADS) xs[c] = c < p.k ? p.h[c] : 0.f;
  __syncthreads();
  while (rp.more()) {
    rp.consume(b0, xs, part, begin);
    rp.load(b0);
    rp.consume(b1, xs, part, begin);
    rp.load(b1);
  }
  __syncthreads();
  for (int i = threadIdx.x; i < end - begin; i += DL_THREADS) {
    const int pair = begin + i, e = pair / p.ff, j = pair - e * p.ff;
    p.act[static_cast<int64_t>(ch.slot[e]) * p.ff + j] = lm_silu(sum_sub(part, 2 * i, ks)) * sum_sub(part, 2 * i + 1, ks);
  }
}

// out[n] = sum over the chosen experts of weight * (down_n . act) + (identity weights) * h[n]: the experts' vectors,
// already multiplied by their weights, stand one after the other in shared memory
__global__ void __launch_bounds__(DL_THREADS, 2) decode_down_kernel(const DecodeExperts p, int ks, int ff_padded) {
  extern __shared__ float dd_smem[];
  __shared__ Chosen ch;
  float* xs = dd_smem;                            // [top][ff_padded]
  float* part = dd_smem + p.r.top * ff_padded;
  // (the choice was made two kernels ago: the kernel before this one has already waited for it)
  read_choice(p, &ch);
  const int pairs = p.k / 2;
  const int begin = static_cast<int>(static_cast<int64_t>(pairs) * blockIdx.x / gridDim.x);
  const int end = static_cast<int>(static_cast<int64_t>(pairs) * (blockIdx.x + 1) / gridDim.x);
  const int lane8 = (threadIdx.x & 31) * 8;
  const int per_expert = ff_padded / DL_PIECE;
  auto addr = [&](int pair, int piece, int r) -> const uint16_t* {
    const int i = piece / per_expert, col = (piece - i * per_expert) * DL_PIECE + lane8;
    if (col >= p.ff) return nullptr;
    return p.down + (static_cast<int64_t>(ch.expert[i]) * p.k + 2 * pair + r) * p.ff + col;
  };
  const int pieces = ch.n * per_expert;
  const int ks_here = pieces < ks ? 1 : ks;
  RowPairs<decltype(addr)> rp(addr, begin, pieces > 0 ? end : begin, pieces, ks_here);
  uint4 b0[DL_UN][2], b1[DL_UN][2];
  rp.load(b0);
  rp.load(b1);
  dependent_wait();
  dependent_trigger();
  for (int i = 0; i < ch.n; ++i)
    for (int c = threadIdx.x; c < ff_padded; c += DL_THREADS)
      xs[i * ff_padded + c] = c < p.ff ? ch.weight[i] * p.act[static_cast<int64_t>(ch.slot[i]) * p.ff + c] : 0.f;
  __syncthreads();
  while (rp.more()) {
    rp.consume(b0, xs, part, begin);
    rp.load(b0);
    rp.consume(b1, xs, part, begin);
    rp.load(b1);
  }
  __syncthreads();
  for (int i = threadIdx.x; i < (end - begin) * 2; i += DL_THREADS) {
    const int row = begin * 2 + i;
    p.out[row] = (pieces > 0 ? sum_sub(part, i, ks_here) : 0.f) + ch.identity * p.h[row];
  }
}

int decode_experts(const DecodeExperts& a, cudaStream_t st) {
  YTC_REQUIRE(a.k % 8 == 0 && a.ff % 8 == 0 && a.r.top <= LM_MAX_TOP, "decode step: bad expert size");
  int s;
  {
    const int pieces = (a.k + DL_PIECE - 1) / DL_PIECE, padded = pieces * DL_PIECE, pairs = a.r.top * a.ff;
    const int grid = pairs < sm_count() ? pairs : sm_count();
    const int per = (pairs + grid - 1) / grid, ks = pick_ks(per, pieces);
    const int smem = (padded + per * 2 * ks) * static_cast<int>(sizeof(float));
    if (smem > 48 * 1024 && (s = ensure_dynamic_smem(reinterpret_cast<const void*>(decode_gate_up_kernel), smem)) != YTC_OK)
      return s;
    YTC_CUDA(launch_overlapped(decode_gate_up_kernel, dim3(grid), dim3(DL_THREADS), smem, st, a, ks, padded));
    count_launch();
    YTC_CUDA(cudaGetLastError());
  }
  const int per_expert = (a.ff + DL_PIECE - 1) / DL_PIECE, ff_padded = per_expert * DL_PIECE, pairs = a.k / 2;
  const int grid = pairs < sm_count() ? pairs : sm_count();
  const int per = (pairs + grid - 1) / grid, ks = pick_ks(per, a.r.top * per_expert);
  const int smem = (a.r.top * ff_padded + per * 2 * ks) * static_cast<int>(sizeof(float));
  if (smem > 220 * 1024) {
    set_last_error("decode step: %d experts of %d channels do not fit shared memory", a.r.top, a.ff);
    return YTC_UNSUPPORTED;
  }
  if (smem > 48 * 1024 && (s = ensure_dynamic_smem(reinterpret_cast<const void*>(decode_down_kernel), smem)) != YTC_OK)
    return s;
  YTC_CUDA(launch_overlapped(decode_down_kernel, dim3(grid), dim3(DL_THREADS), smem, st, a, ks, ff_padded));
  count_launch();
  YTC_CUDA(cudaGetLastError());
  return YTC_OK;
}

}  // namespace ytk
