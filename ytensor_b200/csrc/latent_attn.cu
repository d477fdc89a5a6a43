// Attention over a cache of latents (LatentShape, lm_ops.cuh): what a layer appends to the cache, the rotation, and the form
// for few query rows, in which a head's query is multiplied by its key matrix once, all heads read the cache rows as they
// are, and the value matrix follows the weighted sum. It runs as three kernels: absorb (queries), slices of the cache (16
// heads at a time share every row they read), merge of the slices with the value product. The same kernels serve a decode
// step (fp32 vectors, position read from device memory) and short portions (rows in the model's format).
#include <math_constants.h>

#include <algorithm>

#include "lm_ops.cuh"

namespace ytk {

constexpr int LA_THREADS = 256, LA_WARPS = LA_THREADS / 32;
constexpr int LA_HEADS = 16;       // heads that share a pass over the cache
constexpr int LA_TILE = 64;        // cache rows per step of the tensor-core kernel
constexpr int LA_TILE_SIMT = 32;   // of the FFMA kernel
constexpr int LA_MAX_SPLITS = 64;

template <typename T>
__device__ __forceinline__ float la_load(const void* p, int64_t i) {
  return sizeof(T) == 4 ? static_cast<const float*>(p)[i] : bf16_bits_to_f32(static_cast<const uint16_t*>(p)[i]);
}
template <typename T>
__device__ __forceinline__ void la_store(void* p, int64_t i, float v) {
  if (sizeof(T) == 4) static_cast<float*>(p)[i] = v;
  else static_cast<uint16_t*>(p)[i] = bf16_rn_bits(v);
}
__device__ __forceinline__ void la_cp16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))),
               "l"(src)
               : "memory");
}
__device__ __forceinline__ void la_cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void la_cp_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

// ---------------------------------------------------------------- cache append
// One row by one warp. TI: the projection's format, TC: the cache's.
template <typename TI, typename TC>
__device__ __forceinline__ void append_row(const LatentAppend& p, int row) {
  const int lane = threadIdx.x & 31;
  const int b = row / p.len, t = row - b * p.len;
  const int64_t pos = p.pos ? *p.pos : p.pos0 + t;
  const int64_t in0 = static_cast<int64_t>(row) * p.ld;
  const int64_t out = (static_cast<int64_t>(b) * p.cap + pos) * p.s.row();
  const int64_t c0 = in0 + p.dkv_off, r0 = c0 + p.s.rank;
  // the query latent (unless the caller norms it) and the latent, side by side: pieces of 8 channels
  const TI* in = static_cast<const TI*>(p.in);
  const int q_pieces = p.cq ? p.q_rank / 8 : 0, pieces = q_pieces + p.s.rank / 8;
  float sq = 0.f, sc = 0.f;
#pragma unroll 4
  for (int i = lane; i < pieces; i += 32) {
    const bool is_q = i < q_pieces;
    float v[8];
    Vec8<TI>::load(in + (is_q ? in0 + p.dq_off + i * 8 : c0 + (i - q_pieces) * 8), v);
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) ss = fmaf(v[e], v[e], ss);
    sq += is_q ? ss : 0.f;
    sc += is_q ? 0.f : ss;
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    sq += __shfl_xor_sync(0xffffffffu, sq, o);
    sc += __shfl_xor_sync(0xffffffffu, sc, o);
  }
  const float inv_q = p.cq ? 1.0f / sqrtf(sq / p.q_width + p.eps) : 0.f, inv_c = 1.0f / sqrtf(sc / p.c_width + p.eps);
#pragma unroll 4
  for (int i = lane; i < pieces; i += 32) {
    const bool is_q = i < q_pieces;
    const int e0 = (is_q ? i : i - q_pieces) * 8;
    float v[8], w[8];
    Vec8<TI>::load(in + (is_q ? in0 + p.dq_off : c0) + e0, v);
    Vec8<float>::load((is_q ? p.w_q : p.w_c) + e0, w);
    const float inv = is_q ? inv_q : inv_c;
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] *= inv * w[e];
    if (is_q) Vec8<TI>::store(static_cast<TI*>(p.cq) + static_cast<int64_t>(row) * p.q_rank + e0, v);
    else Vec8<TC>::store(static_cast<TC*>(p.cache) + out + e0, v);
  }
  for (int i = lane; i < p.s.rot / 2; i += 32) {
    float u = la_load<TI>(p.in, r0 + 2 * i), v = la_load<TI>(p.in, r0 + 2 * i + 1);
    if (2 * i < p.s.rot_dims) {
      float sn, cs;
      sincosf(static_cast<float>(pos) * p.s.freq[i], &sn, &cs);
      const float w = u * cs - v * sn;
      v = v * cs + u * sn;
      u = w;
    }
    la_store<TC>(p.cache, out + p.s.rank + 2 * i, u);
    la_store<TC>(p.cache, out + p.s.rank + 2 * i + 1, v);
  }
}

constexpr int AP_WARPS = 4;
template <typename T>
__global__ void __launch_bounds__(AP_WARPS * 32) latent_append_kernel(const LatentAppend p) {
  dependent_wait();
  dependent_trigger();
  const int row = blockIdx.x * AP_WARPS + (threadIdx.x >> 5);
  if (row < p.batch * p.len) append_row<T, T>(p, row);
}

static int check_shape(const LatentShape& s) {
  YTC_REQUIRE(s.heads > 0 && s.dim > 0 && s.dim % 8 == 0 && s.rot >= 0 && s.rot % 16 == 0 && s.rot_dims >= 0 &&
                  s.rot_dims % 2 == 0 && s.rot_dims <= s.rot && s.vdim > 0 && s.vdim % 8 == 0 && s.rank > 0 &&
                  s.rank % 16 == 0 && s.head_ld >= s.dim + s.rot && s.head_ld % 8 == 0 && (s.rot_dims == 0 || s.freq),
              "latent attention: bad sizes");
  return YTC_OK;
}

int latent_append(const LatentAppend& a, cudaStream_t st) {
  int s = check_shape(a.s);
  if (s != YTC_OK) return s;
  YTC_REQUIRE(a.pos || a.pos0 + a.len <= a.cap, "latent_append: the cache is full");
  const int64_t rows = static_cast<int64_t>(a.batch) * a.len;
  YTC_CUDA(launch_overlapped(a.dtype == YTC_BF16 ? latent_append_kernel<uint16_t> : latent_append_kernel<float>,
                             dim3(static_cast<unsigned>((rows + AP_WARPS - 1) / AP_WARPS)), dim3(AP_WARPS * 32), 0, st, a));
  count_launch();
  YTC_CUDA(cudaGetLastError());
  return YTC_OK;
}

// ---------------------------------------------------------------- rotation of the queries
// One row per CTA: the row's sines and cosines once, then every head's pairs.
constexpr int LA_MAX_PAIRS = 128;
template <typename T>
__global__ void __launch_bounds__(128) rotate_queries_kernel(T* q, const LatentShape s, int len, int64_t pos0) {
  __shared__ float sn[LA_MAX_PAIRS], cs[LA_MAX_PAIRS];
  dependent_wait();
  dependent_trigger();
  const int pairs = s.rot_dims / 2;
  const int64_t row = blockIdx.x, pos = pos0 + row % len;
  for (int i = threadIdx.x; i < pairs; i += 128) sincosf(static_cast<float>(pos) * s.freq[i], &sn[i], &cs[i]);
  __syncthreads();
  T* x = q + row * s.heads * s.head_ld + s.dim;
  for (int i = threadIdx.x; i < s.heads * pairs; i += 128) {
    const int h = i / pairs, j = i - h * pairs;
    const int64_t at = static_cast<int64_t>(h) * s.head_ld + 2 * j;
    const float u = la_load<T>(x, at), v = la_load<T>(x, at + 1);
    la_store<T>(x, at, u * cs[j] - v * sn[j]);
    la_store<T>(x, at + 1, v * cs[j] + u * sn[j]);
  }
}

int rotate_queries(void* q, int dtype, const LatentShape& s, int batch, int len, int64_t pos0, cudaStream_t st) {
  const int r = check_shape(s);
  if (r != YTC_OK) return r;
  YTC_REQUIRE(s.rot_dims / 2 <= LA_MAX_PAIRS, "rotate_queries: more than %d rotated dimensions", 2 * LA_MAX_PAIRS);
  if (s.rot_dims == 0) return YTC_OK;
  const dim3 grid(static_cast<unsigned>(static_cast<int64_t>(batch) * len));
  if (dtype == YTC_BF16)
    YTC_CUDA(launch_overlapped(rotate_queries_kernel<uint16_t>, grid, dim3(128), 0, st, static_cast<uint16_t*>(q), s, len, pos0));
  else
    YTC_CUDA(launch_overlapped(rotate_queries_kernel<float>, grid, dim3(128), 0, st, static_cast<float*>(q), s, len, pos0));
  count_launch();
  YTC_CUDA(cudaGetLastError());
  return YTC_OK;
}

// ---------------------------------------------------------------- absorbed queries
// CTA = (row, head, slice of `cols` latent channels): qa[c] = sum over d of q[d] Wk[d][c], eight channels per lane, the
// head's dimensions spread over lanes and warps. The first slice also writes the rotated part. With an append, one more
// CTA per row stores the new cache row.
constexpr int LA_FETCH = 8;  // 16-byte pieces of the matrix a thread requests before it waits for the queries
template <typename TQ, typename TC>
__global__ void __launch_bounds__(LA_THREADS) latent_absorb_kernel(const LatentDecode p, const LatentAppend ap, int cols,
                                                                   int slices) {
  __shared__ float part[LA_WARPS][128];
  __shared__ float q_s[512];
  const LatentShape& s = p.s;
  const int row = blockIdx.y;
  if (static_cast<int>(blockIdx.x) == s.heads * slices) {
    dependent_wait();
    dependent_trigger();
    if (threadIdx.x < 32) append_row<TQ, TC>(ap, row);
    return;
  }
  const int h = blockIdx.x / slices, c0 = (blockIdx.x - h * slices) * cols;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int across = cols / 8, cg = lane % across, dl = lane / across;  // (across divides 32)
  const int groups = LA_WARPS * (32 / across), d0 = warp * (32 / across) + dl;
  const int c = c0 + cg * 8;
  const bool col_ok = c < s.rank;
  const uint16_t* w = p.uk + static_cast<int64_t>(h) * s.dim * s.rank + c;
  uint4 pre[LA_FETCH];
#pragma unroll
  for (int i = 0; i < LA_FETCH; ++i) {
    const int d = d0 + i * groups;
    pre[i] = make_uint4(0u, 0u, 0u, 0u);
    if (col_ok && d < s.dim) pre[i] = *reinterpret_cast<const uint4*>(w + static_cast<int64_t>(d) * s.rank);
  }
  dependent_wait();
  dependent_trigger();
  const int64_t q0 = (static_cast<int64_t>(row) * s.heads + h) * s.head_ld;
  for (int i = threadIdx.x; i < s.dim; i += LA_THREADS) q_s[i] = la_load<TQ>(p.q, q0 + i);
  float* out = p.qa + (static_cast<int64_t>(row) * s.heads + h) * s.row();
  if (c0 == 0) {
    const int64_t pos = p.pos ? *p.pos : p.pos0 + row % p.len;
    for (int i = threadIdx.x; i < s.rot / 2; i += LA_THREADS) {
      float u = la_load<TQ>(p.q, q0 + s.dim + 2 * i), v = la_load<TQ>(p.q, q0 + s.dim + 2 * i + 1);
      if (2 * i < s.rot_dims) {
        float sn, cs;
        sincosf(static_cast<float>(pos) * s.freq[i], &sn, &cs);
        const float t = u * cs - v * sn;
        v = v * cs + u * sn;
        u = t;
      }
      out[s.rank + 2 * i] = u;
      out[s.rank + 2 * i + 1] = v;
    }
  }
  __syncthreads();
  float acc[8] = {};
  auto add = [&](const uint4& u, float x) {
    float f[8];
    Vec8<uint16_t>::unpack(u, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] = fmaf(x, f[e], acc[e]);
  };
#pragma unroll
  for (int i = 0; i < LA_FETCH; ++i)
    if (d0 + i * groups < s.dim) add(pre[i], q_s[d0 + i * groups]);
  for (int d = d0 + LA_FETCH * groups; d < s.dim; d += groups)
    if (col_ok) add(*reinterpret_cast<const uint4*>(w + static_cast<int64_t>(d) * s.rank), q_s[d]);
  for (int o = across; o < 32; o <<= 1)
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], o);
  if (dl == 0)
#pragma unroll
    for (int e = 0; e < 8; ++e) part[warp][cg * 8 + e] = acc[e];
  __syncthreads();
  for (int i = threadIdx.x; i < cols; i += LA_THREADS) {
    if (c0 + i >= s.rank) continue;
    float v = 0.f;
#pragma unroll
    for (int k = 0; k < LA_WARPS; ++k) v += part[k][i];
    out[c0 + i] = v;
  }
}

// ---------------------------------------------------------------- slices of the cache
struct LatentSlice {
  const float* qa;     // [rows][heads][row]
  const void* cache;   // [batch][cap][row]
  float* part;         // [rows][heads][splits][rank + 2]
  const int* pos;
  int64_t cap, pos0;
  int heads, rank, row, len, splits;
  float scale;
};
// Slice `split` of n keys cut into tiles of `tile`: [begin, end); the slices in use are 0 .. used - 1.
__device__ __forceinline__ void slice_of(int64_t n, int tile, int splits, int split, int64_t& begin, int64_t& end, int& used) {
  const int64_t tiles = (n + tile - 1) / tile, per = (tiles + splits - 1) / splits;
  used = static_cast<int>((tiles + per - 1) / per);
  begin = split * per * tile;
  end = begin + per * tile < n ? begin + per * tile : n;
}

__device__ __forceinline__ void la_ldmatrix4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(static_cast<uint32_t>(__cvta_generic_to_shared(p))));
}
__device__ __forceinline__ void la_ldmatrix2(uint32_t (&r)[2], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];"
               : "=r"(r[0]), "=r"(r[1])
               : "r"(static_cast<uint32_t>(__cvta_generic_to_shared(p))));
}
__device__ __forceinline__ void la_ldmatrix2_trans(uint32_t (&r)[2], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];"
               : "=r"(r[0]), "=r"(r[1])
               : "r"(static_cast<uint32_t>(__cvta_generic_to_shared(p))));
}
__device__ __forceinline__ void la_mma(float (&c)[4], const uint32_t (&a)[4], const uint32_t (&b)[2]) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
__device__ __forceinline__ void split_bf16(float v, uint16_t& hi, uint16_t& lo) {
  hi = bf16_rn_bits(v);
  lo = bf16_rn_bits(v - bf16_bits_to_f32(hi));
}

// bf16 cache: 16 heads are the rows of an m16n8k16 product. Queries and weights go in as two bf16 values each (hi + lo, 16
// mantissa bits). Scores: every warp takes 8 of a tile's 64 keys; sums: every warp takes an eighth of the latent channels.
constexpr int LA_NT = 8;  // 8-channel column tiles per warp: up to 512 latent channels
__global__ void __launch_bounds__(LA_THREADS) latent_slice_mma_kernel(const LatentSlice p) {
  extern __shared__ __align__(16) uint8_t la_smem[];
  __shared__ __align__(16) float s_s[LA_HEADS][LA_TILE + 4];
  __shared__ float al_s[LA_HEADS], m_s[LA_HEADS], l_s[LA_HEADS];
  __shared__ __align__(16) uint16_t p_hi[LA_HEADS][LA_TILE + 8], p_lo[LA_HEADS][LA_TILE + 8];
  const int ld = p.row + 8;  // (16 bytes more than a multiple of 32: the rows of an 8 x 8 block lie in different banks)
  uint16_t* q_hi = reinterpret_cast<uint16_t*>(la_smem);
  uint16_t* q_lo = q_hi + LA_HEADS * ld;
  uint16_t* kv = q_lo + LA_HEADS * ld;  // [2][LA_TILE][ld]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int split = blockIdx.x, h0 = blockIdx.y * LA_HEADS, row = blockIdx.z;
  const int nh = p.heads - h0 < LA_HEADS ? p.heads - h0 : LA_HEADS;
  const int64_t pos = p.pos ? *p.pos : p.pos0 + row % p.len;  // (the word was written before this step's first kernel)
  const int64_t n = pos + 1;
  int64_t begin, end;
  int used;
  slice_of(n, LA_TILE, p.splits, split, begin, end, used);
  const uint16_t* cache = static_cast<const uint16_t*>(p.cache) + (row / p.len) * p.cap * p.row;
  const int pieces = p.row / 8;
  // the rows of the tile at key0 before `last`, one row per warp and trip; what lies past `last` is zero
  auto fetch = [&](int64_t key0, int buf, int64_t last) {
    uint16_t* dst = kv + buf * LA_TILE * ld;
#pragma unroll 4
    for (int r = warp; r < LA_TILE; r += LA_WARPS)
      for (int c = lane; c < pieces; c += 32) {
        if (key0 + r < last) la_cp16(dst + r * ld + c * 8, cache + (key0 + r) * p.row + c * 8);
        else *reinterpret_cast<uint4*>(dst + r * ld + c * 8) = make_uint4(0u, 0u, 0u, 0u);
      }
  };
  const int tiles = begin < end ? static_cast<int>((end - begin + LA_TILE - 1) / LA_TILE) : 0;
  // (the newest row may be written by the kernel before this one)
  const int64_t old_end = end < pos ? end : pos;
  if (tiles > 0) fetch(begin, 0, old_end);
  la_cp_commit();
  if (tiles > 1) fetch(begin + LA_TILE, 1, old_end);
  la_cp_commit();
  dependent_wait();
  dependent_trigger();
  if (tiles == 0) return;
  const float* qa = p.qa + (static_cast<int64_t>(row) * p.heads + h0) * p.row;
  for (int h = warp; h < LA_HEADS; h += LA_WARPS)
#pragma unroll 5
    for (int c = lane * 4; c < p.row; c += 128) {
      const float4 v = h < nh ? *reinterpret_cast<const float4*>(qa + h * p.row + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      const uint2 hi = make_uint2(pack_bf16x2_rn(v.x, v.y), pack_bf16x2_rn(v.z, v.w));
      *reinterpret_cast<uint2*>(q_hi + h * ld + c) = hi;
      *reinterpret_cast<uint2*>(q_lo + h * ld + c) =
          make_uint2(pack_bf16x2_rn(v.x - __uint_as_float(hi.x << 16), v.y - __uint_as_float(hi.x & 0xFFFF0000u)),
                     pack_bf16x2_rn(v.z - __uint_as_float(hi.y << 16), v.w - __uint_as_float(hi.y & 0xFFFF0000u)));
    }
  if (threadIdx.x < LA_HEADS) {
    m_s[threadIdx.x] = -CUDART_INF_F;
    l_s[threadIdx.x] = 0.f;
  }
  __syncthreads();  // (zeroes of the requested tiles are in place before the newest row is)
  const int new_tile = pos >= begin && pos < end ? static_cast<int>((pos - begin) / LA_TILE) : -1;
  float acc[LA_NT][4] = {};
  for (int t = 0; t < tiles; ++t) {
    const int buf = t & 1;
    const int64_t key0 = begin + static_cast<int64_t>(t) * LA_TILE;
    uint16_t* tile = kv + buf * LA_TILE * ld;
    la_cp_wait<1>();
    if (t == new_tile && t < 2) {  // (requested above without its newest row)
      const uint16_t* src = cache + pos * p.row;
      for (int c = threadIdx.x; c < pieces; c += LA_THREADS)
        *reinterpret_cast<uint4*>(tile + (pos - key0) * ld + c * 8) = *reinterpret_cast<const uint4*>(src + c * 8);
    }
    __syncthreads();
    {
      float chi[4] = {}, clo[4] = {};
      const uint16_t* b_at = tile + (warp * 8 + (lane & 7)) * ld + ((lane >> 3) & 1) * 8;
      const int a_at = (lane & 15) * ld + (lane >> 4) * 8;
#pragma unroll 4
      for (int k0 = 0; k0 < p.row; k0 += 16) {
        uint32_t ah[4], al[4], b[2];
        la_ldmatrix4(ah, q_hi + a_at + k0);
        la_ldmatrix4(al, q_lo + a_at + k0);
        la_ldmatrix2(b, b_at + k0);
        la_mma(chi, ah, b);
        la_mma(clo, al, b);
      }
      const int r = lane >> 2, c = warp * 8 + (lane & 3) * 2;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int key = c + (e & 1);
        s_s[r + (e >> 1) * 8][key] = key0 + key < end ? (chi[e] + clo[e]) * p.scale : -CUDART_INF_F;
      }
    }
    __syncthreads();
    {  // sixteen lanes per head, four keys each
      const int h = threadIdx.x >> 4, j = threadIdx.x & 15;
      const float4 s4 = *reinterpret_cast<const float4*>(&s_s[h][j * 4]);
      const float s[4] = {s4.x, s4.y, s4.z, s4.w};
      float m = fmaxf(fmaxf(s[0], s[1]), fmaxf(s[2], s[3]));
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
      const float m_old = m_s[h], m_new = fmaxf(m_old, m);  // (every tile has a visible key)
      float l = 0.f;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float w = expf(s[e] - m_new);
        l += w;
        split_bf16(w, p_hi[h][j * 4 + e], p_lo[h][j * 4 + e]);
      }
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
      __syncwarp();
      if (j == 0) {
        const float alpha = expf(m_old - m_new);
        al_s[h] = alpha;
        m_s[h] = m_new;
        l_s[h] = l_s[h] * alpha + l;
      }
    }
    __syncthreads();
    {
      const float a0 = al_s[lane >> 2], a1 = al_s[(lane >> 2) + 8];
#pragma unroll
      for (int i = 0; i < LA_NT; ++i) {
        acc[i][0] *= a0; acc[i][1] *= a0; acc[i][2] *= a1; acc[i][3] *= a1;
      }
#pragma unroll
      for (int kk = 0; kk < LA_TILE / 16; ++kk) {
        uint32_t ah[4], al[4];
        la_ldmatrix4(ah, &p_hi[lane & 15][kk * 16 + (lane >> 4) * 8]);
        la_ldmatrix4(al, &p_lo[lane & 15][kk * 16 + (lane >> 4) * 8]);
#pragma unroll
        for (int i = 0; i < LA_NT; ++i) {
          const int c = (warp + i * LA_WARPS) * 8;
          if (c >= p.rank) break;
          uint32_t b[2];
          la_ldmatrix2_trans(b, tile + (kk * 16 + (lane & 15)) * ld + c);
          la_mma(acc[i], ah, b);
          la_mma(acc[i], al, b);
        }
      }
    }
    __syncthreads();
    if (t + 2 < tiles) fetch(key0 + 2 * LA_TILE, buf, end);
    la_cp_commit();
  }
  const int stride = p.rank + 2;
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int h = (lane >> 2) + half * 8;
    if (h >= nh) continue;
    float* out = p.part + ((static_cast<int64_t>(row) * p.heads + h0 + h) * p.splits + split) * stride;
#pragma unroll
    for (int i = 0; i < LA_NT; ++i) {
      const int c = (warp + i * LA_WARPS) * 8 + (lane & 3) * 2;
      if (c >= p.rank) break;
      *reinterpret_cast<float2*>(out + c) = make_float2(acc[i][half * 2], acc[i][half * 2 + 1]);
    }
  }
  if (threadIdx.x < nh) {
    float* out = p.part + ((static_cast<int64_t>(row) * p.heads + h0 + threadIdx.x) * p.splits + split) * stride + p.rank;
    out[0] = m_s[threadIdx.x];
    out[1] = l_s[threadIdx.x];
  }
}

// The same with fp32 products: a thread computes scores of one key, and sums NC channels of all sixteen heads.
template <typename T, int NC>
__global__ void __launch_bounds__(LA_THREADS) latent_slice_simt_kernel(const LatentSlice p) {
  extern __shared__ __align__(16) uint8_t la_smem[];
  __shared__ float s_s[LA_HEADS][LA_TILE_SIMT + 1], al_s[LA_HEADS], m_s[LA_HEADS], l_s[LA_HEADS];
  const int ld = p.row + 1;
  float* q_s = reinterpret_cast<float*>(la_smem);   // [LA_HEADS][row]
  float* kv = q_s + LA_HEADS * p.row;               // [LA_TILE_SIMT][ld]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int split = blockIdx.x, h0 = blockIdx.y * LA_HEADS, row = blockIdx.z;
  const int nh = p.heads - h0 < LA_HEADS ? p.heads - h0 : LA_HEADS;
  dependent_wait();
  dependent_trigger();
  const int64_t pos = p.pos ? *p.pos : p.pos0 + row % p.len;
  int64_t begin, end;
  int used;
  slice_of(pos + 1, LA_TILE, p.splits, split, begin, end, used);
  if (begin >= end) return;
  const T* cache = static_cast<const T*>(p.cache) + (row / p.len) * p.cap * p.row;
  const float* qa = p.qa + (static_cast<int64_t>(row) * p.heads + h0) * p.row;
  for (int i = threadIdx.x; i < LA_HEADS * p.row; i += LA_THREADS) q_s[i] = i < nh * p.row ? qa[i] : 0.f;
  if (threadIdx.x < LA_HEADS) {
    m_s[threadIdx.x] = -CUDART_INF_F;
    l_s[threadIdx.x] = 0.f;
  }
  float acc[NC][LA_HEADS] = {};
  for (int64_t key0 = begin; key0 < end; key0 += LA_TILE_SIMT) {
    const int keys = end - key0 < LA_TILE_SIMT ? static_cast<int>(end - key0) : LA_TILE_SIMT;
    __syncthreads();
    for (int i = threadIdx.x; i < LA_TILE_SIMT * p.row; i += LA_THREADS) {
      const int r = i / p.row, c = i - r * p.row;
      kv[r * ld + c] = r < keys ? la_load<T>(cache, (key0 + r) * p.row + c) : 0.f;
    }
    __syncthreads();
    for (int h = warp; h < LA_HEADS; h += LA_WARPS) {  // lane = key
      float dot = 0.f;
      for (int c = 0; c < p.row; ++c) dot = fmaf(q_s[h * p.row + c], kv[lane * ld + c], dot);
      const float s = lane < keys ? dot * p.scale : -CUDART_INF_F;
      float m = s;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
      const float m_old = m_s[h], m_new = fmaxf(m_old, m);
      const float w = expf(s - m_new);
      float l = w;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
      s_s[h][lane] = w;
      __syncwarp();
      if (lane == 0) {
        const float alpha = expf(m_old - m_new);
        al_s[h] = alpha;
        m_s[h] = m_new;
        l_s[h] = l_s[h] * alpha + l;
      }
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < NC; ++j) {
      const int c = threadIdx.x + j * LA_THREADS;
      if (c >= p.rank) break;
#pragma unroll
      for (int h = 0; h < LA_HEADS; ++h) acc[j][h] *= al_s[h];
      for (int k = 0; k < keys; ++k) {
        const float v = kv[k * ld + c];
#pragma unroll
        for (int h = 0; h < LA_HEADS; ++h) acc[j][h] = fmaf(s_s[h][k], v, acc[j][h]);
      }
    }
  }
  __syncthreads();
  const int stride = p.rank + 2;
  float* out = p.part + ((static_cast<int64_t>(row) * p.heads + h0) * p.splits + split) * stride;
  const int64_t per_head = static_cast<int64_t>(p.splits) * stride;
#pragma unroll
  for (int j = 0; j < NC; ++j) {
    const int c = threadIdx.x + j * LA_THREADS;
    if (c >= p.rank) break;
#pragma unroll
    for (int h = 0; h < LA_HEADS; ++h)
      if (h < nh) out[h * per_head + c] = acc[j][h];
  }
  if (threadIdx.x < nh) {
    out[threadIdx.x * per_head + p.rank] = m_s[threadIdx.x];
    out[threadIdx.x * per_head + p.rank + 1] = l_s[threadIdx.x];
  }
}

// ---------------------------------------------------------------- merge and value product
// CTA = (row, head, `rows_per` value channels): the head's slices are added up in every CTA, then one warp per channel.
constexpr int LA_VROWS = 16;
template <typename TO>
__global__ void __launch_bounds__(LA_THREADS) latent_values_kernel(const LatentDecode p, int splits, int rows_per, int slices) {
  extern __shared__ __align__(16) uint8_t la_smem[];
  float* ctx = reinterpret_cast<float*>(la_smem);  // [ways][rank]
  __shared__ float w_s[LA_MAX_SPLITS];
  const LatentShape& s = p.s;
  const int row = blockIdx.y, h = blockIdx.x / slices, r0 = (blockIdx.x - h * slices) * rows_per;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const uint16_t* w = p.uv + (static_cast<int64_t>(h) * s.vdim + r0) * s.rank;
  const int here = s.vdim - r0 < rows_per ? s.vdim - r0 : rows_per;
  uint4 pre[LA_VROWS / LA_WARPS][2];  // the first 512 latent channels of this warp's value channels
#pragma unroll
  for (int i = 0; i < LA_VROWS / LA_WARPS; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int r = warp + i * LA_WARPS, c = j * 256 + lane * 8;
      pre[i][j] = make_uint4(0u, 0u, 0u, 0u);
      if (r < here && c < s.rank) pre[i][j] = *reinterpret_cast<const uint4*>(w + static_cast<int64_t>(r) * s.rank + c);
    }
  dependent_wait();
  dependent_trigger();
  const int64_t pos = p.pos ? *p.pos : p.pos0 + row % p.len;
  int64_t begin, end;
  int used;
  slice_of(pos + 1, LA_TILE, splits, 0, begin, end, used);
  const int stride = s.rank + 2;
  const float* part = p.part + (static_cast<int64_t>(row) * s.heads + h) * splits * stride;
  // four channels per thread; threads left over split the slices among them
  const int quads = s.rank / 4, ways = quads < LA_THREADS ? LA_THREADS / quads : 1;
  if (warp == 0) {
    float m[2], l[2], mx = -CUDART_INF_F;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int k = lane + 32 * i;
      m[i] = k < used ? part[k * stride + s.rank] : -CUDART_INF_F;
      l[i] = k < used ? part[k * stride + s.rank + 1] : 0.f;
      mx = fmaxf(mx, m[i]);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      m[i] = expf(m[i] - mx);
      sum = fmaf(m[i], l[i], sum);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
#pragma unroll
    for (int i = 0; i < 2; ++i) w_s[lane + 32 * i] = m[i] / sum;
  }
  __syncthreads();
  for (int q0 = 0; q0 < quads; q0 += LA_THREADS) {
    const int q = q0 + static_cast<int>(threadIdx.x) % (quads < LA_THREADS ? quads : LA_THREADS), way = quads < LA_THREADS ? threadIdx.x / quads : 0;
    if (q >= quads || way >= ways) continue;
    float2 a = make_float2(0.f, 0.f), b = make_float2(0.f, 0.f);
#pragma unroll 8
    for (int k = way; k < used; k += ways) {
      const float w = w_s[k];
      const float2 u = *reinterpret_cast<const float2*>(part + k * stride + q * 4), v = *reinterpret_cast<const float2*>(part + k * stride + q * 4 + 2);
      a.x = fmaf(w, u.x, a.x); a.y = fmaf(w, u.y, a.y);
      b.x = fmaf(w, v.x, b.x); b.y = fmaf(w, v.y, b.y);
    }
    *reinterpret_cast<float4*>(ctx + way * s.rank + q * 4) = make_float4(a.x, a.y, b.x, b.y);
  }
  __syncthreads();
  if (ways > 1) {
    for (int c = threadIdx.x; c < s.rank; c += LA_THREADS) {
      float v = ctx[c];
      for (int k = 1; k < ways; ++k) v += ctx[k * s.rank + c];
      ctx[c] = v;
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < LA_VROWS / LA_WARPS; ++i) {
    const int r = warp + i * LA_WARPS;
    if (r >= here) break;
    float acc = 0.f;
    auto add = [&](const uint4& u, int c) {
      float f[8], x[8];
      Vec8<uint16_t>::unpack(u, f);
      Vec8<float>::load(ctx + c, x);
#pragma unroll
      for (int e = 0; e < 8; ++e) acc = fmaf(x[e], f[e], acc);
    };
#pragma unroll
    for (int j = 0; j < 2; ++j)
      if (j * 256 + lane * 8 < s.rank) add(pre[i][j], j * 256 + lane * 8);
    for (int c = 512 + lane * 8; c < s.rank; c += 256)
      add(*reinterpret_cast<const uint4*>(w + static_cast<int64_t>(r) * s.rank + c), c);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
    if (lane == 0) la_store<TO>(p.out, row * p.ld_out + static_cast<int64_t>(h) * s.vdim + r0 + r, acc);
  }
}

static int latent_splits(int heads, int64_t rows, int64_t max_keys) {
  const int64_t blocks = (heads + LA_HEADS - 1) / LA_HEADS * rows, tiles = (max_keys + LA_TILE - 1) / LA_TILE;
  const int64_t n = std::min<int64_t>(std::min<int64_t>(LA_MAX_SPLITS, tiles), sm_count() / blocks);
  return static_cast<int>(std::max<int64_t>(1, n));
}

int64_t latent_part_floats(const LatentShape& s, int64_t rows, int64_t max_keys) {
  return rows * s.heads * static_cast<int64_t>(latent_splits(s.heads, rows, max_keys)) * (s.rank + 2);
}

int latent_decode(const LatentDecode& a, cudaStream_t st) {
  int r = check_shape(a.s);
  if (r != YTC_OK) return r;
  const LatentShape& s = a.s;
  const int rows = a.batch * a.len;
  YTC_REQUIRE(rows > 0 && rows <= 65535 && a.max_keys > 0 && (!a.pos || rows == 1) && s.dim <= 512 && s.rank <= 1024,
              "latent_decode: head dims up to 512, latents up to 1024 channels");
  const bool q16 = a.io_dtype == YTC_BF16, c16 = a.dtype == YTC_BF16;
  const int sms = sm_count();
  {
    int cols = 64;
    while (cols > 16 && static_cast<int64_t>(s.heads) * ((s.rank + cols - 1) / cols) * rows < sms / 2) cols /= 2;
    const int slices = (s.rank + cols - 1) / cols;
    const dim3 grid(s.heads * slices + (a.append ? 1 : 0), rows);
    const LatentAppend ap = a.append ? *a.append : LatentAppend{};
    auto* fn = q16 ? (c16 ? latent_absorb_kernel<uint16_t, uint16_t> : latent_absorb_kernel<uint16_t, float>)
                   : (c16 ? latent_absorb_kernel<float, uint16_t> : latent_absorb_kernel<float, float>);
    YTC_CUDA(launch_overlapped(fn, grid, dim3(LA_THREADS), 0, st, a, ap, cols, slices));
    count_launch();
    YTC_CUDA(cudaGetLastError());
  }
  const int splits = latent_splits(s.heads, rows, a.max_keys);
  {
    LatentSlice p;
    p.qa = a.qa; p.cache = a.cache; p.part = a.part; p.pos = a.pos;
    p.cap = a.cap; p.pos0 = a.pos0;
    p.heads = s.heads; p.rank = s.rank; p.row = s.row(); p.len = a.len; p.splits = splits;
    p.scale = a.scale;
    const dim3 grid(splits, (s.heads + LA_HEADS - 1) / LA_HEADS, rows);
    void (*fn)(LatentSlice) = nullptr;
    int smem = 0;
    if (c16 && s.rank <= LA_NT * LA_WARPS * 8) {
      fn = latent_slice_mma_kernel;
      smem = (2 * LA_HEADS + 2 * LA_TILE) * (s.row() + 8) * 2;
    } else {
      const int nc = (s.rank + LA_THREADS - 1) / LA_THREADS;
      if (c16) fn = nc <= 1 ? latent_slice_simt_kernel<uint16_t, 1> : nc <= 2 ? latent_slice_simt_kernel<uint16_t, 2> : latent_slice_simt_kernel<uint16_t, 4>;
      else fn = nc <= 1 ? latent_slice_simt_kernel<float, 1> : nc <= 2 ? latent_slice_simt_kernel<float, 2> : latent_slice_simt_kernel<float, 4>;
      smem = (LA_HEADS * s.row() + LA_TILE_SIMT * (s.row() + 1)) * 4;
    }
    if (smem > 216 * 1024) {
      set_last_error("latent_decode: cache rows of %d channels do not fit shared memory", s.row());
      return YTC_UNSUPPORTED;
    }
    if ((r = ensure_dynamic_smem(reinterpret_cast<const void*>(fn), smem)) != YTC_OK) return r;
    YTC_CUDA(launch_overlapped(fn, grid, dim3(LA_THREADS), smem, st, p));
    count_launch();
    YTC_CUDA(cudaGetLastError());
  }
  int rows_per = LA_VROWS;
  while (rows_per > LA_WARPS && static_cast<int64_t>(s.heads) * ((s.vdim + rows_per - 1) / rows_per) * rows < sms / 2) rows_per /= 2;
  const int slices = (s.vdim + rows_per - 1) / rows_per;
  YTC_CUDA(launch_overlapped(q16 ? latent_values_kernel<uint16_t> : latent_values_kernel<float>, dim3(s.heads * slices, rows),
                             dim3(LA_THREADS), std::max(s.rank, 4 * LA_THREADS) * sizeof(float), st, a, splits, rows_per, slices));
  count_launch();
  YTC_CUDA(cudaGetLastError());
  return YTC_OK;
}

}  // namespace ytk

using namespace ytk;

extern "C" int ytcuda_latent_attn_fwd(int dtype, const void* q, const void* uk_bf16, const void* uv_bf16, const void* cache,
                                      int64_t cap, void* out, int batch, int len, int64_t pos0, int heads, int dim, int rot,
                                      int vdim, int rank, const float* freq, float scale, void* stream) {
  YTC_REQUIRE(dtype == YTC_F32 || dtype == YTC_BF16, "ytcuda_latent_attn_fwd: dtype must be fp32 or bf16");
  YTC_REQUIRE(q && uk_bf16 && uv_bf16 && cache && out, "ytcuda_latent_attn_fwd: null argument");
  YTC_REQUIRE(batch > 0 && len > 0 && pos0 >= 0 && pos0 + len <= cap, "ytcuda_latent_attn_fwd: bad extent");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  LatentDecode d;
  d.dtype = d.io_dtype = dtype;
  d.s.heads = heads; d.s.dim = dim; d.s.rot = rot; d.s.vdim = vdim; d.s.head_ld = dim + rot; d.s.rank = rank;
  d.s.rot_dims = rot; d.s.freq = freq;
  d.q = q;
  d.uk = static_cast<const uint16_t*>(uk_bf16); d.uv = static_cast<const uint16_t*>(uv_bf16);
  d.cache = cache; d.cap = cap;
  d.batch = batch; d.len = len; d.pos0 = pos0; d.max_keys = pos0 + len; d.scale = scale;
  d.out = out; d.ld_out = static_cast<int64_t>(heads) * vdim;
  const int64_t rows = static_cast<int64_t>(batch) * len, qa = (rows * heads * (rank + rot) + 3) / 4 * 4;
  auto* ws = static_cast<float*>(device_workspace((qa + latent_part_floats(d.s, rows, d.max_keys)) * sizeof(float), st));
  if (!ws) return YTC_CUDA_ERROR;
  d.qa = ws;
  d.part = ws + qa;
  const int s = latent_decode(d, st);
  device_workspace_release(st);
  return s;
}
