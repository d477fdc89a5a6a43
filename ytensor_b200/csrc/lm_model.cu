// Shared host side of the language models (lm_model.cuh): a call's rows are cut into passes of at most `chunk` tokens per
// sequence and run layer by layer with one launch per operator; one new token of a single sequence runs as a CUDA graph
// of the fused decode kernels, with its position read from device memory, so that one graph serves every step.
#include "lm_model.cuh"

namespace ytk {

LmModel::~LmModel() {
  drop_step();
  if (cap_stream) cudaStreamDestroy(cap_stream);
  for (void* p : pass_owned) cudaFree(p);
  for (void* p : owned) cudaFree(p);
}

bool LmModel::check_config(const char* name) const {
  if (width > 0 && width % 8 == 0 && norm_width > 0 && norm_width <= width && vocab > 0 && batch > 0 && max_tokens > 0 &&
      chunk > 0 && (dtype == YTC_BF16 || dtype == YTC_F32))
    return true;
  set_last_error("%s: unsupported configuration (width must be a multiple of 8, dtype fp32 or bf16)", name);
  return false;
}

int LmModel::alloc_in(std::vector<void*>& list, void** p, int64_t bytes) {
  *p = nullptr;
  if (bytes == 0) return YTC_OK;
  YTC_CUDA(cudaMalloc(p, static_cast<size_t>(bytes)));
  list.push_back(*p);
  return YTC_OK;
}

int LmModel::count_words() const {  // of one layer
  int n = 0;
  for (const MoeLayer* m : moe_layers()) n = std::max(n, m ? m->routes() : 0);
  return n;
}
int LmModel::alloc_counts() { return alloc(count, static_cast<int64_t>(moe_layers().size()) * count_words() * 4); }

int LmModel::ensure_pass(int64_t want_rows) {
  if (want_rows <= rows) return YTC_OK;
  YTC_CUDA(cudaDeviceSynchronize());
  for (void* p : pass_owned) cudaFree(p);
  pass_owned.clear();
  rows = 0;
  const int64_t r = want_rows, w = width, e = esz();
  int64_t ldl = 0, top = 0, tiles = 0, eact = 0, shared = 0;
  for (const MoeLayer* m : moe_layers()) {
    if (!m) continue;
    const int64_t t = moe_max_tiles(r, m->route);
    ldl = std::max<int64_t>(ldl, (m->routes() + 3) / 4 * 4);
    top = std::max<int64_t>(top, m->route.top);
    tiles = std::max(tiles, t);
    eact = std::max<int64_t>(eact, t * LM_GROUP_ROWS * m->ff);
    shared = std::max<int64_t>(shared, m->shared_ff);
  }
  LM_TRY(pass_alloc(x, r * w * 4));
  LM_TRY(pass_alloc(y, r * w * 4));
  LM_TRY(pass_alloc(h, r * w * e));
  LM_TRY(pass_alloc(hf, r * w * e));
  LM_TRY(pass_alloc(ids, r * 4));
  LM_TRY(pass_alloc(want, r * 4));
  LM_TRY(pass_alloc(logit, r * ldl * 4));
  LM_TRY(pass_alloc(choice, r * top * 4));
  LM_TRY(pass_alloc(weight, r * top * 4));
  LM_TRY(pass_alloc(rank, r * top * 4));
  LM_TRY(pass_alloc(slot, r * top * 4));
  LM_TRY(pass_alloc(tile_group, tiles * 4));
  LM_TRY(pass_alloc(grouped, tiles * LM_GROUP_ROWS * w * e));
  LM_TRY(pass_alloc(expert_act, eact * e));
  LM_TRY(pass_alloc(expert_out, tiles * LM_GROUP_ROWS * w * e));
  LM_TRY(pass_alloc(shared_act, r * shared * e));
  // (rows of a block that no token fills are multiplied like the others and never read: they only have to be numbers)
  if (grouped) YTC_CUDA(cudaMemset(grouped, 0, static_cast<size_t>(tiles * LM_GROUP_ROWS * w * e)));
  LM_TRY(alloc_pass(r));
  rows = r;
  return YTC_OK;
}

int LmModel::linear(const void* in, int64_t ldx, const uint16_t* w, void* out, int64_t ldy, int64_t n_rows, int n, int k,
                    LinearEpilogue ex, bool to_f32, cudaStream_t st) const {
  if (bf16()) {
    if (ex.epi == EPI_NONE && !to_f32) ex.epi = EPI_BF16;
    return linear_tc(in, ldx, w, k, out, ldy, to_f32 ? YTC_F32 : YTC_BF16, static_cast<int>(n_rows), n, k, ex, st);
  }
  return linear_f32(static_cast<const float*>(in), ldx, w, k, static_cast<float*>(out), ldy, static_cast<int>(n_rows), n, k,
                    ex, st);
}

ResidualNorm LmModel::residual(int64_t n_rows) const {
  ResidualNorm rn;
  rn.x = x;
  rn.dtype = dtype;
  rn.rows = n_rows;
  rn.width = norm_width;
  rn.ld = width;
  rn.eps = eps;
  rn.h = h;
  rn.h_in = h;
  return rn;
}

int LmModel::clear_counts(cudaStream_t st) {
  if (count) YTC_CUDA(cudaMemsetAsync(count, 0, moe_layers().size() * static_cast<size_t>(count_words()) * sizeof(int), st));
  return YTC_OK;
}

int LmModel::moe_pass(const MoeLayer& m, int layer, int64_t n_rows, ResidualNorm& rn, cudaStream_t st) {
  const int w = width, ldl = (m.routes() + 3) / 4 * 4, tiles = moe_max_tiles(n_rows, m.route), words = count_words();
  int* cnt = count + static_cast<size_t>(layer) * words;
  LM_TRY(linear(h, w, m.router, logit, ldl, n_rows, m.routes(), w, epilogue(EPI_NONE), true, st));
  LM_TRY(moe_route(logit, ldl, m.correction, n_rows, m.route, choice, weight, rank, cnt, st));
  MoeGather g;
  g.h = h; g.dtype = dtype; g.ld = w; g.rows = n_rows; g.r = m.route;
  g.choice = choice; g.rank = rank; g.count = cnt;
  g.grouped = grouped; g.slot = slot; g.tile_group = tile_group; g.n_tiles = tiles;
  if (m.scale_input) {
    g.weight = weight;
    g.x = x;
  }
  LM_TRY(moe_gather(g, st));
  if (m.route.experts > 0) {
    const int64_t gr = static_cast<int64_t>(tiles) * LM_GROUP_ROWS;
    LinearEpilogue up = m.act, down;
    up.tile_group = down.tile_group = tile_group;
    up.groups = down.groups = m.route.experts;
    LM_TRY(linear(grouped, w, m.up, expert_act, m.ff, gr, 2 * m.ff, w, up, false, st));
    LM_TRY(linear(expert_act, m.ff, m.down, expert_out, w, gr, w, m.ff, down, false, st));
  }
  rn.expert_out = expert_out;
  rn.slot = slot;
  rn.weight = m.scale_input ? nullptr : weight;
  rn.top = m.route.top;
  rn.y = nullptr;
  if (m.shared_ff > 0) {
    LM_TRY(linear(h, w, m.shared_up, shared_act, m.shared_ff, n_rows, 2 * m.shared_ff, w, m.shared_act, false, st));
    LM_TRY(linear(shared_act, m.shared_ff, m.shared_down, y, w, n_rows, w, m.shared_ff, epilogue(EPI_NONE), true, st));
    rn.y = y;
  }
  return YTC_OK;
}

int LmModel::logits_of(ResidualNorm rn, const int* want_host, int n_want, float* logits, cudaStream_t st) {
  if (n_want <= 0) return YTC_OK;
  YTC_CUDA(cudaMemcpyAsync(want, want_host, static_cast<size_t>(n_want) * sizeof(int), cudaMemcpyHostToDevice, st));
  rn.w_pre = final_norm;
  rn.row_index = want;
  rn.rows = n_want;
  rn.h = hf;
  LM_TRY(residual_norm(rn, st));
  return linear(hf, width, head, logits, vocab, n_want, vocab, width, epilogue(EPI_NONE), true, st);
}

// ------------------------------------------------------------------ decode step
__global__ void set_word_kernel(int* p, int v) { *p = v; }

DecodeInput LmModel::step_input(const float* w_pre) {
  DecodeInput in;
  in.width = norm_width;
  in.eps = eps;
  in.w_pre = w_pre;
  if (step_post) {
    in.kind = DECODE_RESIDUAL;
    in.x_in = sx[step_cur];
    in.y = sy;
    in.w_post = step_post;
    step_cur ^= 1;
    in.x_out = sx[step_cur];
  } else {
    in.kind = DECODE_EMBED;
    in.id = step_id;
    in.embed = embed;
    in.vocab = vocab;
    in.embed_scale = embed_scale;
    in.x_out = sx[step_cur];
  }
  return in;
}

DecodeInput LmModel::step_plain(const float* v) {
  DecodeInput in;
  in.plain = v;
  return in;
}

int LmModel::step_linear(const DecodeInput& in, const uint16_t* w, int n, int k, const LinearEpilogue& ex, float* out,
                         int* advance, cudaStream_t st) const {
  DecodeLinear a;
  a.in = in;
  a.w = w; a.n = n; a.k = k; a.ex = ex; a.out = out; a.advance = advance;
  return decode_linear(a, st);
}

int LmModel::step_moe(const MoeLayer& m, const float* w_pre, cudaStream_t st) {
  DecodeRoute r;
  r.in = step_input(w_pre);
  r.w = m.router; r.correction = m.correction; r.k = width; r.r = m.route;
  r.h = sh; r.choice = step_choice; r.weight = step_weight;
  LM_TRY(decode_route(r, st));
  DecodeExperts e;
  e.gate_up = m.up; e.down = m.down; e.k = width; e.ff = m.ff; e.r = m.route;
  e.act = m.act; e.scale_input = m.scale_input;
  e.shared_gate_up = m.shared_up; e.shared_down = m.shared_down; e.shared_ff = m.shared_ff; e.shared_act = m.shared_act;
  e.choice = step_choice; e.weight = step_weight; e.h = sh; e.mid = sact; e.out = sy;
  return decode_experts(e, st);
}

int LmModel::ensure_step() {
  if (pos) return YTC_OK;
  int64_t act = std::max(1, step_act_floats());
  for (const MoeLayer* m : moe_layers())
    if (m) act = std::max<int64_t>(act, static_cast<int64_t>(m->route.top) * m->ff + m->shared_ff);
  LM_TRY(alloc(sx[0], width * 4));
  LM_TRY(alloc(sx[1], width * 4));
  LM_TRY(alloc(sy, width * 4));
  LM_TRY(alloc(sh, width * 4));
  LM_TRY(alloc(sact, act * 4));
  LM_TRY(alloc(step_choice, LM_MAX_TOP * 4));
  LM_TRY(alloc(step_weight, LM_MAX_TOP * 4));
  LM_TRY(alloc(step_logits, static_cast<int64_t>(vocab) * 4));
  LM_TRY(alloc(step_id, 16));
  LM_TRY(alloc_step());
  YTC_CUDA(cudaStreamCreateWithFlags(&cap_stream, cudaStreamNonBlocking));
  return alloc(pos, 16);
}

void LmModel::drop_step() {
  if (step) cudaGraphExecDestroy(step);
  step = nullptr;
  step_ready = false;
}

int LmModel::build_step() {
  drop_step();
  const uint64_t before = ytcuda_launch_count();
  YTC_CUDA(cudaStreamBeginCapture(cap_stream, cudaStreamCaptureModeThreadLocal));
  step_begin();
  const int s = step_launches(cap_stream);
  cudaGraph_t graph = nullptr;
  const cudaError_t e = cudaStreamEndCapture(cap_stream, &graph);
  step_kernels = static_cast<int>(ytcuda_launch_count() - before);
  if (s != YTC_OK) {
    if (graph) cudaGraphDestroy(graph);
    cudaGetLastError();
    return s;
  }
  YTC_CUDA(e);
  const cudaError_t i = cudaGraphInstantiate(&step, graph, 0);
  cudaGraphDestroy(graph);
  YTC_CUDA(i);
  step_ready = true;
  return YTC_OK;
}

// One token of the one sequence through the graph.
int LmModel::run_step(const int* id, bool wanted, float* logits, cudaStream_t st) {
  LM_TRY(ensure_step());
  if (!step_ready) LM_TRY(build_step());
  if (dev_pos != len) {
    set_word_kernel<<<1, 1, 0, st>>>(pos, static_cast<int>(len));
    count_launch();
    YTC_CUDA(cudaGetLastError());
  }
  YTC_CUDA(cudaMemcpyAsync(step_id, id, sizeof(int), cudaMemcpyDeviceToDevice, st));
  dev_pos = -1;
  YTC_CUDA(cudaGraphLaunch(step, st));
  count_launch(static_cast<uint64_t>(step_kernels));
  dev_pos = len + 1;
  if (wanted)
    YTC_CUDA(cudaMemcpyAsync(logits, step_logits, static_cast<size_t>(vocab) * sizeof(float), cudaMemcpyDeviceToDevice, st));
  return YTC_OK;
}

// ------------------------------------------------------------------ calls
bool LmModel::set_common_weight(const std::string& n, const void* p) {
  drop_step();
  if (n == "embed") embed = static_cast<const uint16_t*>(p);
  else if (n == "head") head = static_cast<const uint16_t*>(p);
  else if (n == "norm") final_norm = static_cast<const float*>(p);
  else return false;
  return true;
}

int LmModel::reset() {
  len = 0;
  return clear_state();
}

int LmModel::forward(const int32_t* tokens, int n, const int32_t* wanted, int n_want, float* logits, cudaStream_t st) {
  OverlapGuard overlap_guard;
  YTC_REQUIRE(tokens, "forward: null argument");
  YTC_REQUIRE(n > 0 && n_want >= 0 && (n_want == 0 || (wanted && logits)), "forward: bad arguments");
  YTC_REQUIRE(len + n <= max_tokens, "forward: %lld tokens do not fit a sequence of at most %d",
              static_cast<long long>(len + n), max_tokens);
  YTC_REQUIRE(embed && head && final_norm, "forward: embed / head / norm not set");
  YTC_REQUIRE(weights_set(), "forward: a layer weight is not set");
  const int B = batch;
  for (int i = 0; i < n_want; ++i)
    YTC_REQUIRE(wanted[i] >= 0 && wanted[i] < static_cast<int64_t>(B) * n, "forward: wanted row %d out of range", wanted[i]);
  if (B == 1 && n == 1 && decode_path == 0) {
    LM_TRY(run_step(tokens, n_want > 0, logits, st));
    for (int i = 1; i < n_want; ++i)
      YTC_CUDA(cudaMemcpyAsync(logits + static_cast<int64_t>(i) * vocab, logits, static_cast<size_t>(vocab) * 4,
                               cudaMemcpyDeviceToDevice, st));
    len += 1;
    return YTC_OK;
  }
  const int most = std::min(n, chunk);
  LM_TRY(ensure_pass(static_cast<int64_t>(B) * most));
  for (int t0 = 0; t0 < n; t0 += most) {
    const int m = std::min(most, n - t0);
    const int32_t* pass_ids = tokens + t0;
    if (B > 1 && m < n) {  // the pass's columns of the id matrix
      YTC_CUDA(cudaMemcpy2DAsync(ids, static_cast<size_t>(m) * 4, tokens + t0, static_cast<size_t>(n) * 4,
                                 static_cast<size_t>(m) * 4, B, cudaMemcpyDeviceToDevice, st));
      pass_ids = ids;
    }
    // wanted rows that lie in this pass, in runs of consecutive places of the output
    std::vector<int> pass_rows, place;
    for (int i = 0; i < n_want; ++i) {
      const int b = wanted[i] / n, t = wanted[i] - b * n;
      if (t >= t0 && t < t0 + m) {
        pass_rows.push_back(b * m + t - t0);
        place.push_back(i);
      }
    }
    bool run = true;
    for (size_t i = 1; i < place.size(); ++i) run = run && place[i] == place[0] + static_cast<int>(i);
    if (pass_rows.size() > static_cast<size_t>(rows)) run = false;
    YTC_REQUIRE(run, "forward: wanted rows must be distinct and, when the call is longer than %d tokens, in the order of the "
                "tokens", chunk);
    LM_TRY(pass(pass_ids, m, pass_rows.data(), static_cast<int>(pass_rows.size()),
                pass_rows.empty() ? nullptr : logits + static_cast<int64_t>(place[0]) * vocab, st));
    len += m;
  }
  return YTC_OK;
}

}  // namespace ytk

using namespace ytk;

extern "C" {

// ---------------------------------------------------------------- any model's handle
void ytcuda_lm_destroy(void* handle) {
  auto* m = static_cast<LmModel*>(handle);
  if (!m) return;
  cudaDeviceSynchronize();
  delete m;
}

int ytcuda_lm_reset(void* handle) {
  auto* m = static_cast<LmModel*>(handle);
  YTC_REQUIRE(m, "ytcuda_lm_reset: null handle");
  return m->reset();
}

int64_t ytcuda_lm_cache_len(void* handle) {
  auto* m = static_cast<LmModel*>(handle);
  return m ? m->len : -1;
}

int ytcuda_lm_set_decode_path(void* handle, int path) {
  auto* m = static_cast<LmModel*>(handle);
  YTC_REQUIRE(m, "ytcuda_lm_set_decode_path: null handle");
  YTC_REQUIRE(path == 0 || path == 1, "ytcuda_lm_set_decode_path: path must be 0 or 1");
  m->decode_path = path;
  return YTC_OK;
}

int ytcuda_lm_forward(void* handle, const int32_t* ids, int len, const int32_t* want, int n_want, float* logits,
                      void* stream) {
  auto* m = static_cast<LmModel*>(handle);
  YTC_REQUIRE(m, "ytcuda_lm_forward: null handle");
  return m->forward(ids, len, want, n_want, logits, static_cast<cudaStream_t>(stream));
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
                     int identity, int top, int groups, int keep, int score, int32_t* choice, float* weight, int32_t* rank,
                     int32_t* count, void* stream) {
  YTC_REQUIRE(rows >= 0 && (rows == 0 || (logits && choice && weight && rank && count)), "ytcuda_moe_route: null argument");
  YTC_REQUIRE(score == ROUTE_SOFTMAX || score == ROUTE_SIGMOID, "ytcuda_moe_route: unknown score");
  return moe_route(logits, row_stride, correction, rows, RouterSpec{experts, identity, top, groups, keep, score}, choice,
                   weight, rank, count, static_cast<cudaStream_t>(stream));
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
                      int64_t y_row_stride, int m, int n, int k, int act_cols, float limit, const int32_t* block_group,
                      int groups, void* stream) {
  YTC_REQUIRE(dtype == YTC_F32 || dtype == YTC_BF16, "ytcuda_linear_act: dtype must be fp32 or bf16");
  YTC_REQUIRE(act >= 0 && act <= 5 && m >= 0 && n >= 0 && k > 0 && groups >= 1, "ytcuda_linear_act: bad argument");
  YTC_REQUIRE(x && w_bf16 && y, "ytcuda_linear_act: null argument");
  static const int kinds[] = {EPI_NONE, EPI_GELU_ERF, EPI_SWIGLU_PAIRS, EPI_RELU2, EPI_SILU, EPI_CLAMP_PAIRS};
  LinearEpilogue ex;
  ex.epi = act == 0 && dtype == YTC_BF16 ? static_cast<int>(EPI_BF16) : kinds[act];
  ex.act_cols = act_cols;
  ex.limit = limit;
  ex.tile_group = block_group;
  ex.groups = groups;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (dtype == YTC_BF16) return linear_tc(x, x_row_stride, w_bf16, k, y, y_row_stride, YTC_BF16, m, n, k, ex, st);
  return linear_f32(static_cast<const float*>(x), x_row_stride, static_cast<const uint16_t*>(w_bf16), k,
                    static_cast<float*>(y), y_row_stride, m, n, k, ex, st);
}

int ytcuda_gated_rows(int dtype, const void* in, int64_t in_stride, const void* gate, int64_t gate_stride, void* out,
                      int64_t out_stride, int64_t rows, int cols, int width, const float* w, float eps, void* stream) {
  YTC_REQUIRE(dtype == YTC_F32 || dtype == YTC_BF16, "ytcuda_gated_rows: dtype must be fp32 or bf16");
  YTC_REQUIRE(in && gate && out, "ytcuda_gated_rows: null argument");
  GatedRows a;
  a.dtype = dtype;
  a.in = in; a.gate = gate; a.out = out;
  a.ld_in = in_stride; a.ld_gate = gate_stride; a.ld_out = out_stride;
  a.rows = rows; a.cols = cols; a.width = width; a.w = w; a.eps = eps;
  return gated_rows(a, static_cast<cudaStream_t>(stream));
}

}  // extern "C"
