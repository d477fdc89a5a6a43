// Duzozen decoder-only language model: per layer a norm before and after each sublayer, sliding-window attention with
// capped scores and no rotation, values mixed with the first mixing layer's, and a dense or mixture-of-experts
// feed-forward. This file is the model's host side: weights, K/V rings, buffers and the order of launches. The mechanisms
// are in lm_ops.cuh (window_attention, append_kv, residual_norm, linear_tc / linear_f32, moe_*, decode_*).
//
// Several tokens per call run layer by layer with one launch per operator (tensor-core linears in bf16, FFMA linears in
// fp32); the rows of a call are cut into passes of at most `chunk` tokens per sequence, so that a window's ring holds
// window - 1 + chunk positions however long the sequence is. One new token of a single sequence runs as a CUDA graph of
// the fused decode kernels; the position is read from device memory, so one graph serves every step.
#include <algorithm>
#include <cstring>
#include <string>
#include <vector>

#include "lm_ops.cuh"

namespace ytk {

struct DuzozenLayer {
  ytcuda_duzozen_layer c{};
  const float *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr, *vmix = nullptr,
              *correction = nullptr;
  const uint16_t *qkv = nullptr, *o = nullptr, *up = nullptr, *down = nullptr, *router = nullptr;
  int qkv_w = 0, att_w = 0, mix = VMIX_NONE;
  int ring = 0;
  void *k = nullptr, *v = nullptr;  // [batch][kv_heads][ring][dim / vdim]
  RouterSpec route() const { return RouterSpec{c.experts, c.identity, c.top, c.groups, c.keep}; }
};

struct DuzozenModel {
  ytcuda_duzozen_config c{};
  std::vector<DuzozenLayer> layers;
  const uint16_t *embed = nullptr, *head = nullptr;
  const float* final_norm = nullptr;
  int64_t len = 0;        // tokens in every sequence
  int decode_path = 0;    // 0: the graph of fused kernels for one token of one sequence, 1: the operator path always
  std::vector<void*> owned;
  // buffers of a pass of `rows` rows
  int64_t rows = 0;
  std::vector<void*> pass_owned;
  float *x = nullptr, *y = nullptr, *logit = nullptr, *weight = nullptr;
  void *h = nullptr, *hf = nullptr, *qkv = nullptr, *att = nullptr, *act = nullptr, *v_first = nullptr,
       *grouped = nullptr, *expert_act = nullptr, *expert_out = nullptr;
  int *ids = nullptr, *want = nullptr, *choice = nullptr, *rank = nullptr, *slot = nullptr, *tile_group = nullptr,
      *count = nullptr;
  // decode step
  bool step_ready = false;
  int64_t dev_pos = -1;   // what the position word on the device holds
  int *pos = nullptr, *step_id = nullptr, *step_choice = nullptr;
  float *sx[2] = {}, *sy = nullptr, *sqkv = nullptr, *satt = nullptr, *sact = nullptr, *sh = nullptr, *sv_first = nullptr,
        *step_weight = nullptr, *step_logits = nullptr;
  cudaStream_t cap_stream = nullptr;
  cudaGraphExec_t step = nullptr;
  int step_kernels = 0;

  bool bf16() const { return c.dtype == YTC_BF16; }
  int esz() const { return bf16() ? 2 : 4; }
  int max_routes() const {
    int n = 0;
    for (const DuzozenLayer& L : layers) n = std::max(n, L.c.mlp == YTC_MLP_MOE ? L.c.experts + L.c.identity : 0);
    return n;
  }
};

static int dz_alloc(std::vector<void*>& owned, void** p, size_t bytes) {
  *p = nullptr;
  if (bytes == 0) return YTC_OK;
  YTC_CUDA(cudaMalloc(p, bytes));
  owned.push_back(*p);
  return YTC_OK;
}
#define DZ_ALLOC(owned, field, bytes)                                                          \
  do {                                                                                         \
    const int _s = dz_alloc(owned, reinterpret_cast<void**>(&m->field), static_cast<size_t>(bytes)); \
    if (_s != YTC_OK) return _s;                                                               \
  } while (0)
#define DZ(expr)                     \
  do {                               \
    const int _s = (expr);           \
    if (_s != YTC_OK) return _s;     \
  } while (0)

static int ensure_pass(DuzozenModel* m, int64_t rows) {
  if (rows <= m->rows) return YTC_OK;
  YTC_CUDA(cudaDeviceSynchronize());
  for (void* p : m->pass_owned) cudaFree(p);
  m->pass_owned.clear();
  m->rows = 0;
  const int64_t w = m->c.width;
  int64_t qkv = 0, att = 0, act = 0, vf = 0, logit = 0, top = 0, tiles = 0, eact = 0;
  for (const DuzozenLayer& L : m->layers) {
    qkv = std::max<int64_t>(qkv, L.qkv_w);
    att = std::max<int64_t>(att, L.att_w);
    if (L.mix != VMIX_NONE) vf = std::max<int64_t>(vf, static_cast<int64_t>(L.c.kv_heads) * L.c.vdim);
    if (L.c.mlp == YTC_MLP_DENSE) act = std::max<int64_t>(act, L.c.ff);
    if (L.c.mlp == YTC_MLP_MOE) {
      const int64_t t = moe_max_tiles(rows, L.route());
      logit = std::max<int64_t>(logit, (L.c.experts + L.c.identity + 3) / 4 * 4);
      top = std::max<int64_t>(top, L.c.top);
      tiles = std::max(tiles, t);
      eact = std::max<int64_t>(eact, t * LM_GROUP_ROWS * L.c.ff);
    }
  }
  const int64_t e = m->esz();
  std::vector<void*>& o = m->pass_owned;
  DZ_ALLOC(o, x, rows * w * 4);
  DZ_ALLOC(o, y, rows * w * 4);
  DZ_ALLOC(o, h, rows * w * e);
  DZ_ALLOC(o, hf, rows * w * e);
  DZ_ALLOC(o, qkv, rows * qkv * e);
  DZ_ALLOC(o, att, rows * att * e);
  DZ_ALLOC(o, act, rows * act * e);
  DZ_ALLOC(o, v_first, rows * vf * e);
  DZ_ALLOC(o, ids, rows * 4);
  DZ_ALLOC(o, want, rows * 4);
  DZ_ALLOC(o, logit, rows * logit * 4);
  DZ_ALLOC(o, choice, rows * top * 4);
  DZ_ALLOC(o, weight, rows * top * 4);
  DZ_ALLOC(o, rank, rows * top * 4);
  DZ_ALLOC(o, slot, rows * top * 4);
  DZ_ALLOC(o, tile_group, tiles * 4);
  DZ_ALLOC(o, grouped, tiles * LM_GROUP_ROWS * w * e);
  DZ_ALLOC(o, expert_act, eact * e);
  DZ_ALLOC(o, expert_out, tiles * LM_GROUP_ROWS * w * e);
  // (rows of a block that no token fills are multiplied like the others and never read: they only have to be numbers)
  if (m->grouped) YTC_CUDA(cudaMemset(m->grouped, 0, tiles * LM_GROUP_ROWS * w * e));
  m->rows = rows;
  return YTC_OK;
}

// y = epilogue(x . W^T): activations in the model's type, y in it too (to_f32: fp32).
static int dz_linear(DuzozenModel* m, const void* x, int64_t ldx, const uint16_t* w, void* y, int64_t ldy, int64_t rows,
                     int n, int k, int epi, bool to_f32, cudaStream_t st, const int* tile_group = nullptr, int groups = 1) {
  LinearEpilogue ex;
  ex.tile_group = tile_group;
  ex.groups = groups;
  if (m->bf16()) {
    ex.epi = (epi == EPI_NONE && !to_f32) ? EPI_BF16 : epi;
    return linear_tc(x, ldx, w, k, y, ldy, to_f32 ? YTC_F32 : YTC_BF16, static_cast<int>(rows), n, k, ex, st);
  }
  ex.epi = epi;
  return linear_f32(static_cast<const float*>(x), ldx, w, k, static_cast<float*>(y), ldy, static_cast<int>(rows), n, k, ex, st);
}

// One pass over `len` tokens per sequence at positions m->len ..: ids [batch][len] on the device. `want` / n_want: rows
// of the pass whose logits go to `logits` [n_want][vocab].
static int dz_pass(DuzozenModel* m, const int* ids, int len, const int* want, int n_want, float* logits, cudaStream_t st) {
  const int B = m->c.batch, w = m->c.width;
  const int64_t rows = static_cast<int64_t>(B) * len;
  DZ(ytcuda_embedding(m->embed, ids, m->x, rows, w, m->c.vocab, st));
  const int routes = m->max_routes();
  if (routes > 0) YTC_CUDA(cudaMemsetAsync(m->count, 0, m->layers.size() * static_cast<size_t>(routes) * sizeof(int), st));
  ResidualNorm rn;  // what the next residual kernel adds to the stream: the sublayer before it
  rn.x = m->x;
  rn.dtype = m->c.dtype;
  rn.rows = rows;
  rn.width = m->c.norm_width;
  rn.ld = w;
  rn.eps = m->c.eps;
  rn.h = m->h;
  rn.h_in = m->h;
  for (size_t l = 0; l < m->layers.size(); ++l) {
    const DuzozenLayer& L = m->layers[l];
    const ytcuda_duzozen_layer& c = L.c;
    rn.w_pre = L.norm1;
    DZ(residual_norm(rn, st));
    DZ(dz_linear(m, m->h, w, L.qkv, m->qkv, L.qkv_w, rows, L.qkv_w, w, EPI_NONE, false, st));
    AppendKv ap;
    ap.dtype = m->c.dtype;
    ap.qkv = m->qkv; ap.ld = L.qkv_w;
    ap.k_off = c.heads * c.dim; ap.v_off = (c.heads + c.kv_heads) * c.dim;
    ap.k = L.k; ap.v = L.v;
    ap.v_first = m->v_first; ap.lambda = L.vmix; ap.mix = L.mix;
    ap.batch = B; ap.len = len; ap.kv_heads = c.kv_heads; ap.dim = c.dim; ap.vdim = c.vdim; ap.ring = L.ring;
    ap.pos0 = m->len;
    DZ(append_kv(ap, st));
    WindowAttn at;
    at.dtype = m->c.dtype;
    at.q = m->qkv; at.k = L.k; at.v = L.v; at.o = m->att;
    at.batch = B; at.kv_heads = c.kv_heads; at.groups = c.heads / c.kv_heads; at.q_len = len;
    at.head_dim = c.dim; at.value_dim = c.vdim;
    at.q_st[0] = static_cast<int64_t>(len) * L.qkv_w; at.q_st[1] = c.dim; at.q_st[2] = L.qkv_w;
    at.k_st[0] = static_cast<int64_t>(c.kv_heads) * L.ring * c.dim; at.k_st[1] = static_cast<int64_t>(L.ring) * c.dim; at.k_st[2] = c.dim;
    at.v_st[0] = static_cast<int64_t>(c.kv_heads) * L.ring * c.vdim; at.v_st[1] = static_cast<int64_t>(L.ring) * c.vdim; at.v_st[2] = c.vdim;
    at.o_st[0] = static_cast<int64_t>(len) * L.att_w; at.o_st[1] = c.vdim; at.o_st[2] = L.att_w;
    at.pos0 = m->len; at.window = c.window; at.ring = L.ring;
    at.scale = c.scale; at.softcap = c.softcap;
    DZ(window_attention(at, st));
    DZ(dz_linear(m, m->att, L.att_w, L.o, m->y, w, rows, w, L.att_w, EPI_NONE, true, st));
    rn.y = m->y;
    rn.slot = nullptr;
    rn.w_post = L.norm1b;
    if (c.mlp == YTC_MLP_NONE) continue;
    rn.w_pre = L.norm2;
    DZ(residual_norm(rn, st));
    rn.w_post = L.norm2b;
    if (c.mlp == YTC_MLP_DENSE) {
      DZ(dz_linear(m, m->h, w, L.up, m->act, c.ff, rows, c.ff, w, EPI_GELU_ERF, false, st));
      DZ(dz_linear(m, m->act, c.ff, L.down, m->y, w, rows, w, c.ff, EPI_NONE, true, st));
      continue;
    }
    const RouterSpec r = L.route();
    const int n_routes = c.experts + c.identity, ldl = (n_routes + 3) / 4 * 4, tiles = moe_max_tiles(rows, r);
    int* count = m->count + l * static_cast<size_t>(routes);
    DZ(dz_linear(m, m->h, w, L.router, m->logit, ldl, rows, n_routes, w, EPI_NONE, true, st));
    DZ(moe_route(m->logit, ldl, L.correction, rows, r, m->choice, m->weight, m->rank, count, st));
    DZ(moe_gather(m->h, m->c.dtype, w, rows, r, m->choice, m->rank, count, m->grouped, m->slot, m->tile_group, tiles, st));
    if (c.experts > 0) {
      const int64_t gr = static_cast<int64_t>(tiles) * LM_GROUP_ROWS;
      DZ(dz_linear(m, m->grouped, w, L.up, m->expert_act, c.ff, gr, 2 * c.ff, w, EPI_SWIGLU_PAIRS, false, st, m->tile_group,
                   c.experts));
      DZ(dz_linear(m, m->expert_act, c.ff, L.down, m->expert_out, w, gr, w, c.ff, EPI_NONE, false, st, m->tile_group,
                   c.experts));
    }
    rn.expert_out = m->expert_out;
    rn.slot = m->slot;
    rn.weight = m->weight;
    rn.top = c.top;
  }
  if (n_want > 0) {  // only the wanted rows go through the last residual sum, the final norm and the vocabulary matrix
    YTC_CUDA(cudaMemcpyAsync(m->want, want, static_cast<size_t>(n_want) * sizeof(int), cudaMemcpyHostToDevice, st));
    rn.w_pre = m->final_norm;
    rn.row_index = m->want;
    rn.rows = n_want;
    rn.h = m->hf;
    DZ(residual_norm(rn, st));
    DZ(dz_linear(m, m->hf, w, m->head, logits, m->c.vocab, n_want, m->c.vocab, w, EPI_NONE, true, st));
  }
  return YTC_OK;
}

// ------------------------------------------------------------------ decode step
__global__ void set_word_kernel(int* p, int v) { *p = v; }

static int ensure_step(DuzozenModel* m) {
  if (m->pos) return YTC_OK;
  const int64_t w = m->c.width;
  int64_t qkv = 0, att = 0, act = 1, vf = 1;
  for (const DuzozenLayer& L : m->layers) {
    qkv = std::max<int64_t>(qkv, L.qkv_w);
    att = std::max<int64_t>(att, L.att_w);
    vf = std::max<int64_t>(vf, static_cast<int64_t>(L.c.kv_heads) * L.c.vdim);
    if (L.c.mlp == YTC_MLP_DENSE) act = std::max<int64_t>(act, L.c.ff);
    if (L.c.mlp == YTC_MLP_MOE) act = std::max<int64_t>(act, static_cast<int64_t>(L.c.top) * L.c.ff);
  }
  std::vector<void*>& o = m->owned;
  DZ_ALLOC(o, sx[0], w * 4);
  DZ_ALLOC(o, sx[1], w * 4);
  DZ_ALLOC(o, sy, w * 4);
  DZ_ALLOC(o, sqkv, qkv * 4);
  DZ_ALLOC(o, satt, att * 4);
  DZ_ALLOC(o, sact, act * 4);
  DZ_ALLOC(o, sh, w * 4);
  DZ_ALLOC(o, sv_first, vf * 4);
  DZ_ALLOC(o, step_choice, LM_MAX_TOP * 4);
  DZ_ALLOC(o, step_weight, LM_MAX_TOP * 4);
  DZ_ALLOC(o, step_logits, static_cast<int64_t>(m->c.vocab) * 4);
  DZ_ALLOC(o, step_id, 16);
  YTC_CUDA(cudaStreamCreateWithFlags(&m->cap_stream, cudaStreamNonBlocking));
  DZ_ALLOC(o, pos, 16);
  return YTC_OK;
}

static int dz_step_launches(DuzozenModel* m, cudaStream_t st) {
  const int w = m->c.width;
  int cur = 0;                 // sx[cur] holds the residual row
  const float* w_post = nullptr;  // norm behind the sublayer whose output is in sy (null: nothing to add yet)
  auto input = [&](const float* w_pre) {
    DecodeInput in;
    in.width = m->c.norm_width;
    in.eps = m->c.eps;
    in.w_pre = w_pre;
    if (w_post) {
      in.kind = 1;
      in.x_in = m->sx[cur];
      in.y = m->sy;
      in.w_post = w_post;
      cur ^= 1;
      in.x_out = m->sx[cur];
    } else {
      in.kind = 0;
      in.id = m->step_id;
      in.embed = m->embed;
      in.vocab = m->c.vocab;
      in.x_out = m->sx[cur];
    }
    return in;
  };
  auto linear = [&](const DecodeInput& in, const uint16_t* wt, int n, int k, int epi, float* out, int* advance) {
    DecodeLinear a;
    a.in = in;
    a.w = wt; a.n = n; a.k = k; a.epi = epi; a.out = out; a.advance = advance;
    return decode_linear(a, st);
  };
  auto plain = [&](const float* v) {
    DecodeInput in;
    in.plain = v;
    return in;
  };
  for (const DuzozenLayer& L : m->layers) {
    const ytcuda_duzozen_layer& c = L.c;
    DZ(linear(input(L.norm1), L.qkv, L.qkv_w, w, EPI_NONE, m->sqkv, nullptr));
    DecodeAttn at;
    at.dtype = m->c.dtype;
    at.qkv = m->sqkv; at.k = L.k; at.v = L.v; at.v_first = m->sv_first; at.lambda = L.vmix; at.mix = L.mix;
    at.out = m->satt; at.pos = m->pos;
    at.kv_heads = c.kv_heads; at.groups = c.heads / c.kv_heads; at.dim = c.dim; at.vdim = c.vdim;
    at.ring = L.ring; at.window = c.window;
    at.max_keys = c.window > 0 ? std::min<int64_t>(c.window, m->c.max_tokens) : m->c.max_tokens;
    at.scale = c.scale; at.softcap = c.softcap;
    DZ(decode_attention(at, st));
    DZ(linear(plain(m->satt), L.o, w, L.att_w, EPI_NONE, m->sy, nullptr));
    w_post = L.norm1b;
    if (c.mlp == YTC_MLP_NONE) continue;
    if (c.mlp == YTC_MLP_DENSE) {
      DZ(linear(input(L.norm2), L.up, c.ff, w, EPI_GELU_ERF, m->sact, nullptr));
      DZ(linear(plain(m->sact), L.down, w, c.ff, EPI_NONE, m->sy, nullptr));
    } else {
      DecodeRoute r;
      r.in = input(L.norm2);
      r.w = L.router; r.correction = L.correction; r.k = w; r.r = L.route();
      r.h = m->sh; r.choice = m->step_choice; r.weight = m->step_weight;
      DZ(decode_route(r, st));
      DecodeExperts e;
      e.gate_up = L.up; e.down = L.down; e.k = w; e.ff = c.ff; e.r = L.route();
      e.choice = m->step_choice; e.weight = m->step_weight; e.h = m->sh; e.act = m->sact; e.out = m->sy;
      DZ(decode_experts(e, st));
    }
    w_post = L.norm2b;
  }
  return linear(input(m->final_norm), m->head, m->c.vocab, w, EPI_NONE, m->step_logits, m->pos);
}

static void drop_step(DuzozenModel* m) {
  if (m->step) cudaGraphExecDestroy(m->step);
  m->step = nullptr;
  m->step_ready = false;
}

static int build_step(DuzozenModel* m) {
  drop_step(m);
  const uint64_t before = ytcuda_launch_count();
  YTC_CUDA(cudaStreamBeginCapture(m->cap_stream, cudaStreamCaptureModeThreadLocal));
  const int s = dz_step_launches(m, m->cap_stream);
  cudaGraph_t graph = nullptr;
  const cudaError_t e = cudaStreamEndCapture(m->cap_stream, &graph);
  m->step_kernels = static_cast<int>(ytcuda_launch_count() - before);
  if (s != YTC_OK) {
    if (graph) cudaGraphDestroy(graph);
    cudaGetLastError();
    return s;
  }
  YTC_CUDA(e);
  const cudaError_t i = cudaGraphInstantiate(&m->step, graph, 0);
  cudaGraphDestroy(graph);
  YTC_CUDA(i);
  m->step_ready = true;
  return YTC_OK;
}

// One token of the one sequence through the graph.
static int dz_step(DuzozenModel* m, const int* id, bool want, float* logits, cudaStream_t st) {
  DZ(ensure_step(m));
  if (!m->step_ready) DZ(build_step(m));
  if (m->dev_pos != m->len) {
    set_word_kernel<<<1, 1, 0, st>>>(m->pos, static_cast<int>(m->len));
    count_launch();
    YTC_CUDA(cudaGetLastError());
  }
  YTC_CUDA(cudaMemcpyAsync(m->step_id, id, sizeof(int), cudaMemcpyDeviceToDevice, st));
  m->dev_pos = -1;
  YTC_CUDA(cudaGraphLaunch(m->step, st));
  count_launch(static_cast<uint64_t>(m->step_kernels));
  m->dev_pos = m->len + 1;
  if (want)
    YTC_CUDA(cudaMemcpyAsync(logits, m->step_logits, static_cast<size_t>(m->c.vocab) * sizeof(float),
                             cudaMemcpyDeviceToDevice, st));
  return YTC_OK;
}

static bool step_applies(const DuzozenModel* m, int len) { return m->c.batch == 1 && len == 1 && m->decode_path == 0; }

static void dz_free(DuzozenModel* m) {
  drop_step(m);
  if (m->cap_stream) cudaStreamDestroy(m->cap_stream);
  for (void* p : m->pass_owned) cudaFree(p);
  for (void* p : m->owned) cudaFree(p);
  delete m;
}

static bool bad_layer(const ytcuda_duzozen_layer& c, std::string* why) {
  auto fail = [&](const char* t) {
    *why = t;
    return true;
  };
  if (c.heads <= 0 || c.kv_heads <= 0 || c.heads % c.kv_heads) return fail("heads must be a multiple of kv_heads");
  if (c.dim <= 0 || c.dim % 8 || c.vdim <= 0 || c.vdim % 8 || c.dim > 256 || c.vdim > 256)
    return fail("head dims must be multiples of 8, at most 256");
  if (c.window < 0 || c.softcap < 0.f) return fail("negative window or softcap");
  if (c.mlp < YTC_MLP_NONE || c.mlp > YTC_MLP_MOE) return fail("unknown feed-forward kind");
  if (c.mlp != YTC_MLP_NONE && (c.ff <= 0 || c.ff % 8)) return fail("the feed-forward width must be a multiple of 8");
  if (c.mlp == YTC_MLP_MOE) {
    const int n = c.experts + c.identity;
    if (c.experts < 0 || c.identity < 0 || n <= 0 || n > LM_MAX_ROUTES) return fail("bad number of experts");
    if (c.top <= 0 || c.top > n || c.top > LM_MAX_TOP) return fail("bad number of chosen experts");
    if (c.groups <= 0 || n % c.groups || c.keep <= 0 || c.keep > c.groups) return fail("bad expert groups");
  }
  return false;
}

}  // namespace ytk

using namespace ytk;

extern "C" {

void* ytcuda_duzozen_create(const ytcuda_duzozen_config* cfg, const ytcuda_duzozen_layer* layers) {
  if (!cfg || !layers || cfg->layers <= 0 || cfg->width <= 0 || cfg->width % 8 || cfg->norm_width <= 0 ||
      cfg->norm_width > cfg->width || cfg->vocab <= 0 || cfg->batch <= 0 || cfg->max_tokens <= 0 || cfg->chunk <= 0 ||
      (cfg->dtype != YTC_BF16 && cfg->dtype != YTC_F32)) {
    set_last_error("ytcuda_duzozen_create: unsupported configuration (width must be a multiple of 8, dtype fp32 or bf16)");
    return nullptr;
  }
  auto* m = new DuzozenModel();
  m->c = *cfg;
  m->c.chunk = std::min(cfg->chunk, cfg->max_tokens);
  bool first_seen = false;
  int vf = 0;
  for (int l = 0; l < cfg->layers; ++l) {
    DuzozenLayer L;
    L.c = layers[l];
    std::string why;
    if (bad_layer(L.c, &why)) {
      set_last_error("ytcuda_duzozen_create: layer %d: %s", l, why.c_str());
      delete m;
      return nullptr;
    }
    L.qkv_w = (L.c.heads + L.c.kv_heads) * L.c.dim + L.c.kv_heads * L.c.vdim;
    L.att_w = L.c.heads * L.c.vdim;
    if (L.c.v_mix) {
      const int mine = L.c.kv_heads * L.c.vdim;
      if (first_seen && mine != vf) {
        set_last_error("ytcuda_duzozen_create: layer %d mixes values of another size than the first mixing layer's", l);
        delete m;
        return nullptr;
      }
      L.mix = first_seen ? VMIX_MIX : VMIX_FIRST;
      first_seen = true;
      vf = mine;
    }
    // Rings are whole tiles of 128 positions. A pass of `chunk` tokens needs the window before its first token and
    // itself, wherever these fall between tile borders.
    auto tile = [](int64_t n) { return (n + 127) / 128 * 128; };
    int64_t ring = tile(m->c.max_tokens);
    if (L.c.window > 0) ring = std::min(ring, tile(static_cast<int64_t>(L.c.window) - 1 + m->c.chunk) + 128);
    L.ring = static_cast<int>(ring);
    m->layers.push_back(L);
  }
  bool ok = true;
  const size_t routes = static_cast<size_t>(m->max_routes());
  if (routes) ok = dz_alloc(m->owned, reinterpret_cast<void**>(&m->count), m->layers.size() * routes * sizeof(int)) == YTC_OK;
  for (DuzozenLayer& L : m->layers) {
    const size_t kb = static_cast<size_t>(cfg->batch) * L.c.kv_heads * L.ring * L.c.dim * m->esz();
    const size_t vb = static_cast<size_t>(cfg->batch) * L.c.kv_heads * L.ring * L.c.vdim * m->esz();
    ok = ok && dz_alloc(m->owned, &L.k, kb) == YTC_OK && dz_alloc(m->owned, &L.v, vb) == YTC_OK &&
         cudaMemset(L.k, 0, kb) == cudaSuccess && cudaMemset(L.v, 0, vb) == cudaSuccess;
  }
  if (!ok) {
    set_last_error("ytcuda_duzozen_create: device allocation failed");
    dz_free(m);
    return nullptr;
  }
  return m;
}

void ytcuda_duzozen_destroy(void* handle) {
  auto* m = static_cast<DuzozenModel*>(handle);
  if (!m) return;
  cudaDeviceSynchronize();
  dz_free(m);
}

int ytcuda_duzozen_set_weight(void* handle, const char* name, int layer, const void* dptr) {
  auto* m = static_cast<DuzozenModel*>(handle);
  YTC_REQUIRE(m && name && dptr, "ytcuda_duzozen_set_weight: null argument");
  YTC_REQUIRE((reinterpret_cast<uint64_t>(dptr) & 15) == 0, "ytcuda_duzozen_set_weight: weights must be 16-byte aligned");
  const std::string n(name);
  const auto* f = static_cast<const float*>(dptr);
  const auto* b = static_cast<const uint16_t*>(dptr);
  drop_step(m);
  if (n == "embed") { m->embed = b; return YTC_OK; }
  if (n == "head") { m->head = b; return YTC_OK; }
  if (n == "norm") { m->final_norm = f; return YTC_OK; }
  YTC_REQUIRE(layer >= 0 && layer < m->c.layers, "ytcuda_duzozen_set_weight: layer %d out of range", layer);
  DuzozenLayer& L = m->layers[layer];
  if (n == "norm1") L.norm1 = f;
  else if (n == "norm1b") L.norm1b = f;
  else if (n == "norm2") L.norm2 = f;
  else if (n == "norm2b") L.norm2b = f;
  else if (n == "vmix") L.vmix = f;
  else if (n == "correction") L.correction = f;
  else if (n == "qkv") L.qkv = b;
  else if (n == "o") L.o = b;
  else if (n == "up") L.up = b;
  else if (n == "down") L.down = b;
  else if (n == "router") L.router = b;
  else {
    set_last_error("ytcuda_duzozen_set_weight: unknown weight name '%s'", name);
    return YTC_INVALID_ARG;
  }
  return YTC_OK;
}

int ytcuda_duzozen_reset(void* handle) {
  auto* m = static_cast<DuzozenModel*>(handle);
  YTC_REQUIRE(m, "ytcuda_duzozen_reset: null handle");
  m->len = 0;
  return YTC_OK;
}

int64_t ytcuda_duzozen_cache_len(void* handle) {
  auto* m = static_cast<DuzozenModel*>(handle);
  return m ? m->len : -1;
}

int ytcuda_duzozen_set_decode_path(void* handle, int path) {
  auto* m = static_cast<DuzozenModel*>(handle);
  YTC_REQUIRE(m, "ytcuda_duzozen_set_decode_path: null handle");
  YTC_REQUIRE(path == 0 || path == 1, "ytcuda_duzozen_set_decode_path: path must be 0 or 1");
  m->decode_path = path;
  return YTC_OK;
}

int ytcuda_duzozen_forward(void* handle, const int32_t* ids, int len, const int32_t* want, int n_want, float* logits,
                           void* stream) {
  struct OverlapGuard {
    OverlapGuard() { overlap_scope() = true; }
    ~OverlapGuard() { overlap_scope() = false; }
  } overlap_guard;
  auto* m = static_cast<DuzozenModel*>(handle);
  YTC_REQUIRE(m && ids, "ytcuda_duzozen_forward: null argument");
  YTC_REQUIRE(len > 0 && n_want >= 0 && (n_want == 0 || (want && logits)), "ytcuda_duzozen_forward: bad arguments");
  YTC_REQUIRE(m->len + len <= m->c.max_tokens, "ytcuda_duzozen_forward: %lld tokens do not fit a sequence of at most %d",
              static_cast<long long>(m->len + len), m->c.max_tokens);
  YTC_REQUIRE(m->embed && m->head && m->final_norm, "ytcuda_duzozen_forward: embed / head / norm not set");
  for (const DuzozenLayer& L : m->layers) {
    bool ok = L.norm1 && L.norm1b && L.qkv && L.o && (L.mix != VMIX_MIX || L.vmix);
    if (L.c.mlp != YTC_MLP_NONE) ok = ok && L.norm2 && L.norm2b;
    if (L.c.mlp == YTC_MLP_DENSE) ok = ok && L.up && L.down;
    if (L.c.mlp == YTC_MLP_MOE) ok = ok && L.router && L.correction && (L.c.experts == 0 || (L.up && L.down));
    YTC_REQUIRE(ok, "ytcuda_duzozen_forward: a layer weight is not set");
  }
  const int B = m->c.batch;
  for (int i = 0; i < n_want; ++i)
    YTC_REQUIRE(want[i] >= 0 && want[i] < static_cast<int64_t>(B) * len, "ytcuda_duzozen_forward: wanted row %d out of range",
                want[i]);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (step_applies(m, len)) {
    DZ(dz_step(m, ids, n_want > 0, logits, st));
    for (int i = 1; i < n_want; ++i)
      YTC_CUDA(cudaMemcpyAsync(logits + static_cast<int64_t>(i) * m->c.vocab, logits, static_cast<size_t>(m->c.vocab) * 4,
                               cudaMemcpyDeviceToDevice, st));
    m->len += 1;
    return YTC_OK;
  }
  const int most = std::min(len, m->c.chunk);
  DZ(ensure_pass(m, static_cast<int64_t>(B) * most));
  for (int t0 = 0; t0 < len; t0 += most) {
    const int n = std::min(most, len - t0);
    const int32_t* pass_ids = ids + t0;
    if (B > 1 && n < len) {  // the pass's columns of the id matrix
      YTC_CUDA(cudaMemcpy2DAsync(m->ids, static_cast<size_t>(n) * 4, ids + t0, static_cast<size_t>(len) * 4,
                                 static_cast<size_t>(n) * 4, B, cudaMemcpyDeviceToDevice, st));
      pass_ids = m->ids;
    }
    // wanted rows that lie in this pass, in runs of consecutive places of the output
    std::vector<int> rows;
    std::vector<int> place;
    for (int i = 0; i < n_want; ++i) {
      const int b = want[i] / len, t = want[i] - b * len;
      if (t >= t0 && t < t0 + n) {
        rows.push_back(b * n + t - t0);
        place.push_back(i);
      }
    }
    bool run = true;
    for (size_t i = 1; i < place.size(); ++i) run = run && place[i] == place[0] + static_cast<int>(i);
    if (rows.size() > static_cast<size_t>(m->rows)) run = false;
    YTC_REQUIRE(run, "ytcuda_duzozen_forward: wanted rows must be distinct and, when the call is longer than %d tokens, in "
                "the order of the tokens", m->c.chunk);
    DZ(dz_pass(m, pass_ids, n, rows.data(), static_cast<int>(rows.size()),
               rows.empty() ? nullptr : logits + static_cast<int64_t>(place[0]) * m->c.vocab, st));
    m->len += n;
  }
  return YTC_OK;
}

// ---------------------------------------------------------------- single mechanisms
int ytcuda_window_attn_fwd(int dtype, const void* q, const void* k, const void* v, void* o, int batch, int kv_heads,
                           int groups, int q_len, int head_dim, int value_dim, const int64_t* q_strides,
                           const int64_t* k_strides, const int64_t* v_strides, const int64_t* o_strides, int64_t pos0,
                           int window, int ring, float scale, float softcap, void* stream) {
  YTC_REQUIRE(dtype == YTC_F32 || dtype == YTC_BF16, "ytcuda_window_attn_fwd: dtype must be fp32 or bf16");
  YTC_REQUIRE(q && k && v && o && q_strides && k_strides && v_strides && o_strides, "ytcuda_window_attn_fwd: null argument");
  YTC_REQUIRE(pos0 >= 0 && head_dim > 0 && value_dim > 0 && softcap >= 0.f, "ytcuda_window_attn_fwd: bad argument");
  WindowAttn a;
  a.dtype = dtype;
  a.q = q; a.k = k; a.v = v; a.o = o;
  a.batch = batch; a.kv_heads = kv_heads; a.groups = groups; a.q_len = q_len; a.head_dim = head_dim; a.value_dim = value_dim;
  for (int i = 0; i < 3; ++i) {
    a.q_st[i] = q_strides[i];
    a.k_st[i] = k_strides[i];
    a.v_st[i] = v_strides[i];
    a.o_st[i] = o_strides[i];
  }
  a.pos0 = pos0; a.window = window; a.ring = ring; a.scale = scale; a.softcap = softcap;
  return window_attention(a, static_cast<cudaStream_t>(stream));
}

int ytcuda_moe_route(const float* logits, int64_t row_stride, const float* correction, int64_t rows, int experts,
                     int identity, int top, int groups, int keep, int32_t* choice, float* weight, int32_t* rank,
                     int32_t* count, void* stream) {
  YTC_REQUIRE(rows >= 0 && (rows == 0 || (logits && correction && choice && weight && rank && count)),
              "ytcuda_moe_route: null argument");
  return moe_route(logits, row_stride, correction, rows, RouterSpec{experts, identity, top, groups, keep}, choice, weight,
                   rank, count, static_cast<cudaStream_t>(stream));
}

int ytcuda_residual_norm(float* x, const float* y, const float* w_post, const float* w_pre, void* h, int dtype, int64_t rows,
                         int width, int row_stride, float eps, void* stream) {
  YTC_REQUIRE(dtype == YTC_F32 || dtype == YTC_BF16, "ytcuda_residual_norm: dtype must be fp32 or bf16");
  YTC_REQUIRE(x && (!w_post || y) && (!w_pre || h), "ytcuda_residual_norm: null argument");
  ResidualNorm a;
  a.x = x; a.y = y; a.w_post = w_post; a.w_pre = w_pre; a.h = h; a.dtype = dtype;
  a.rows = rows; a.width = width; a.ld = row_stride; a.eps = eps;
  return residual_norm(a, static_cast<cudaStream_t>(stream));
}

int ytcuda_linear_act(int dtype, int act, const void* x, int64_t x_row_stride, const void* w_bf16, void* y,
                      int64_t y_row_stride, int m, int n, int k, const int32_t* block_group, int groups, void* stream) {
  YTC_REQUIRE(dtype == YTC_F32 || dtype == YTC_BF16, "ytcuda_linear_act: dtype must be fp32 or bf16");
  YTC_REQUIRE(act >= 0 && act <= 2 && m >= 0 && n >= 0 && k > 0 && groups >= 1, "ytcuda_linear_act: bad argument");
  YTC_REQUIRE(x && w_bf16 && y, "ytcuda_linear_act: null argument");
  LinearEpilogue ex;
  ex.epi = act == 0 ? (dtype == YTC_BF16 ? EPI_BF16 : EPI_NONE) : act == 1 ? EPI_GELU_ERF : EPI_SWIGLU_PAIRS;
  ex.tile_group = block_group;
  ex.groups = groups;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (dtype == YTC_BF16) return linear_tc(x, x_row_stride, w_bf16, k, y, y_row_stride, YTC_BF16, m, n, k, ex, st);
  return linear_f32(static_cast<const float*>(x), x_row_stride, static_cast<const uint16_t*>(w_bf16), k,
                    static_cast<float*>(y), y_row_stride, m, n, k, ex, st);
}

}  // extern "C"
