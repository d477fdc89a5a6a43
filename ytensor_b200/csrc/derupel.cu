// Derupel decoder-only language model: sublayers read the residual stream itself and are normed on their output only; the
// mixers are linear attention with a decayed state per head and causal attention over cached latents with a rotated key
// part shared by the heads, both with an output gate; the feed-forwards are dense (squared relu) or a mixture of experts
// (bounded gates, sigmoid router whose weights multiply the experts' inputs, a shared expert), or none. This file is the
// model's own host side: weights, latent caches, states, buffers and the order of launches; passes, decode graph and
// experts are LmModel's (lm_model.cuh), the mechanisms are in lm_ops.cuh (latent_*, decayed_attention, gated_rows, ...).
#include "lm_model.cuh"

namespace ytk {

struct DerupelLayer {
  ytcuda_derupel_layer c{};
  const float *norm1 = nullptr, *norm2 = nullptr, *mix_norm = nullptr, *decay = nullptr, *dq_norm = nullptr,
              *dkv_norm = nullptr;
  const uint16_t *in = nullptr, *o = nullptr, *uq = nullptr, *uk = nullptr, *uv = nullptr, *expand = nullptr, *up = nullptr,
                 *down = nullptr;
  LatentShape latent;
  MoeLayer moe;
  int in_w = 0, att_w = 0;     // fused input projection, concatenated heads
  int gate_off = 0;            // columns of the projection that hold the output gate
  float* state = nullptr;      // [batch][heads][dim][vdim]
  void* cache = nullptr;       // [batch][max_tokens][rank + rot]
  bool is_latent() const { return c.mixer == YTC_MIXER_LATENT; }
  int q_w() const { return c.heads * c.head_ld; }
  int expand_w() const { return c.heads * (c.head_ld + c.vdim); }
};

struct DerupelModel : LmModel {
  std::vector<DerupelLayer> layers;
  void *proj = nullptr, *cq = nullptr, *q = nullptr, *att = nullptr, *act = nullptr;  // of a pass
  float *qa = nullptr, *part = nullptr;
  void* expanded = nullptr;   // keys and values of one layer, [batch][positions][heads * (head_ld + vdim)]
  int64_t expanded_rows = 0;  // positions it holds
  float *sproj = nullptr, *sq = nullptr, *satt = nullptr, *sqa = nullptr, *spart = nullptr;  // of a decode step

  ~DerupelModel() override { cudaFree(expanded); }
  template <typename F>
  int64_t widest(F f) const {
    int64_t n = 0;
    for (const DerupelLayer& L : layers) n = std::max<int64_t>(n, f(L));
    return n;
  }
  int step_act_floats() const override {  // (of the dense layers)
    return static_cast<int>(widest([](const DerupelLayer& L) { return L.c.mlp == YTC_MLP_DENSE ? L.c.ff : 0; }));
  }
  std::vector<const MoeLayer*> moe_layers() const override {
    std::vector<const MoeLayer*> v;
    for (const DerupelLayer& L : layers) v.push_back(L.c.mlp == YTC_MLP_MOE ? &L.moe : nullptr);
    return v;
  }
  int64_t proj_width() const { return widest([](const DerupelLayer& L) { return L.in_w; }); }
  int64_t att_width() const { return widest([](const DerupelLayer& L) { return L.att_w; }); }
  int64_t q_width() const { return widest([](const DerupelLayer& L) { return L.is_latent() ? L.q_w() : 0; }); }
  int64_t qa_floats(int64_t r) const {
    return widest([&](const DerupelLayer& L) { return L.is_latent() ? r * L.c.heads * L.latent.row() : 0; });
  }
  int64_t part_floats(int64_t r) const {
    return widest([&](const DerupelLayer& L) { return L.is_latent() ? latent_part_floats(L.latent, r, max_tokens) : 0; });
  }
  int alloc_pass(int64_t r) override {
    const int64_t e = esz(), few = std::min<int64_t>(r, LATENT_MAX_ROWS);
    int64_t parts = 0;
    for (int64_t i = 1; i <= few; ++i) parts = std::max(parts, part_floats(i));
    LM_TRY(pass_alloc(proj, r * proj_width() * e));
    LM_TRY(pass_alloc(cq, r * widest([](const DerupelLayer& L) { return L.c.q_rank; }) * e));
    LM_TRY(pass_alloc(q, r * q_width() * e));
    LM_TRY(pass_alloc(att, r * att_width() * e));
    LM_TRY(pass_alloc(act, r * step_act_floats() * e));
    LM_TRY(pass_alloc(qa, qa_floats(few) * 4));
    return pass_alloc(part, parts * 4);
  }
  int alloc_step() override {
    LM_TRY(alloc(sproj, proj_width() * 4));
    LM_TRY(alloc(sq, q_width() * 4));
    LM_TRY(alloc(satt, att_width() * 4));
    LM_TRY(alloc(sqa, qa_floats(1) * 4));
    return alloc(spart, part_floats(1) * 4);
  }
  bool weights_set() const override {
    for (const DerupelLayer& L : layers) {
      bool ok = L.norm1 && L.in && L.o;
      if (L.is_latent()) ok = ok && L.uq && L.uk && L.uv && L.expand && L.dq_norm && L.dkv_norm && (L.c.rot_dims == 0 || L.latent.freq);
      else ok = ok && L.mix_norm && L.decay;
      if (L.c.mlp != YTC_MLP_NONE) ok = ok && L.norm2;
      if (L.c.mlp == YTC_MLP_DENSE) ok = ok && L.up && L.down;
      if (L.c.mlp == YTC_MLP_MOE)
        ok = ok && L.moe.router && L.moe.up && L.moe.down && (L.c.shared_ff == 0 || (L.moe.shared_up && L.moe.shared_down));
      if (!ok) return false;
    }
    return true;
  }
  int ensure_expanded(int64_t positions);
  int mix_latent(const DerupelLayer& L, int n, cudaStream_t st);
  int mix_decayed(const DerupelLayer& L, int n, cudaStream_t st);
  int pass(const int* ids, int n, const int* want, int n_want, float* logits, cudaStream_t st) override;
  LatentAppend append_of(const DerupelLayer& L) const;
  int step_latent(const DerupelLayer& L, cudaStream_t st);
  int step_decayed(const DerupelLayer& L, cudaStream_t st);
  int step_launches(cudaStream_t st) override;
};

// Room for the expanded keys and values of `positions` positions, grown in large pieces. Rows behind the newest position are
// masked by the attention but still multiplied: everything in the buffer has to be a number.
int DerupelModel::ensure_expanded(int64_t positions) {
  if (positions <= expanded_rows) return YTC_OK;
  YTC_CUDA(cudaDeviceSynchronize());
  cudaFree(expanded);
  expanded = nullptr;
  expanded_rows = 0;
  const int64_t most = (max_tokens + 127) / 128 * 128;
  const int64_t n = std::max(positions, std::min<int64_t>(most, (positions + 4095) / 4096 * 4096));
  const int64_t bytes = batch * n * widest([](const DerupelLayer& L) { return L.is_latent() ? L.expand_w() : 0; }) * esz();
  YTC_CUDA(cudaMalloc(&expanded, static_cast<size_t>(bytes)));
  YTC_CUDA(cudaMemset(expanded, 0, static_cast<size_t>(bytes)));
  YTC_CUDA(cudaDeviceSynchronize());
  expanded_rows = n;
  return YTC_OK;
}

LatentAppend DerupelModel::append_of(const DerupelLayer& L) const {
  LatentAppend a;
  a.dtype = dtype;
  a.s = L.latent;
  a.ld = L.in_w;
  a.dq_off = 0; a.dkv_off = L.c.q_rank; a.q_rank = L.c.q_rank;
  a.q_width = L.c.q_width; a.c_width = L.c.c_width;
  a.w_q = L.dq_norm; a.w_c = L.dkv_norm;
  a.eps = eps;
  a.cache = L.cache;
  a.cap = max_tokens;
  return a;
}

// h -> att: [query latent; latent, rotated key part; gate], cache, queries, attention, gate
int DerupelModel::mix_latent(const DerupelLayer& L, int n, cudaStream_t st) {
  const ytcuda_derupel_layer& c = L.c;
  const int64_t n_rows = static_cast<int64_t>(batch) * n;
  LM_TRY(linear(h, width, L.in, proj, L.in_w, n_rows, L.in_w, width, epilogue(EPI_NONE), false, st));
  LatentAppend ap = append_of(L);
  ap.in = proj; ap.cq = cq;
  ap.batch = batch; ap.len = n; ap.pos0 = len;
  LM_TRY(latent_append(ap, st));
  LM_TRY(linear(cq, c.q_rank, L.uq, q, L.q_w(), n_rows, L.q_w(), c.q_rank, epilogue(EPI_NONE), false, st));
  if (n_rows <= LATENT_MAX_ROWS) {
    LatentDecode d;
    d.dtype = d.io_dtype = dtype;
    d.s = L.latent;
    d.q = q; d.uk = L.uk; d.uv = L.uv; d.cache = L.cache; d.cap = max_tokens;
    d.batch = batch; d.len = n; d.pos0 = len; d.max_keys = max_tokens; d.scale = c.scale;
    d.qa = qa; d.part = part; d.out = att; d.ld_out = L.att_w;
    LM_TRY(latent_decode(d, st));
  } else {
    const int64_t end = len + n, ring = (end + 127) / 128 * 128, ew = L.expand_w();
    LM_TRY(ensure_expanded(ring));
    LM_TRY(rotate_queries(q, dtype, L.latent, batch, n, len, st));
    for (int b = 0; b < batch; ++b)
      LM_TRY(linear(static_cast<const char*>(L.cache) + static_cast<int64_t>(b) * max_tokens * L.latent.row() * esz(),
                    L.latent.row(), L.expand, static_cast<char*>(expanded) + b * ring * ew * esz(), ew, end,
                    static_cast<int>(ew), L.latent.row(), epilogue(EPI_NONE), false, st));
    WindowAttn at;
    at.dtype = dtype;
    at.q = q; at.k = expanded; at.v = static_cast<const char*>(expanded) + static_cast<int64_t>(L.q_w()) * esz(); at.o = att;
    at.batch = batch; at.kv_heads = c.heads; at.groups = 1; at.q_len = n;
    at.head_dim = c.head_ld; at.value_dim = c.vdim;
    at.q_st[0] = static_cast<int64_t>(n) * L.q_w(); at.q_st[1] = c.head_ld; at.q_st[2] = L.q_w();
    at.k_st[0] = ring * ew; at.k_st[1] = c.head_ld; at.k_st[2] = ew;
    at.v_st[0] = ring * ew; at.v_st[1] = c.vdim; at.v_st[2] = ew;
    at.o_st[0] = static_cast<int64_t>(n) * L.att_w; at.o_st[1] = c.vdim; at.o_st[2] = L.att_w;
    at.pos0 = len; at.window = 0; at.ring = static_cast<int>(ring);
    at.scale = c.scale; at.softcap = 0.f;
    LM_TRY(window_attention(at, st));
  }
  GatedRows g;
  g.dtype = dtype;
  g.in = g.out = att; g.ld_in = g.ld_out = L.att_w;
  g.gate = static_cast<const char*>(proj) + static_cast<int64_t>(L.gate_off) * esz(); g.ld_gate = L.in_w;
  g.rows = n_rows; g.cols = L.att_w;
  return gated_rows(g, st);
}

// h -> att: [queries, keys, values; gate], state, norm and gate
int DerupelModel::mix_decayed(const DerupelLayer& L, int n, cudaStream_t st) {
  const ytcuda_derupel_layer& c = L.c;
  const int64_t n_rows = static_cast<int64_t>(batch) * n;
  LinearEpilogue silu = epilogue(EPI_SILU);
  silu.act_cols = L.gate_off;
  LM_TRY(linear(h, width, L.in, proj, L.in_w, n_rows, L.in_w, width, silu, false, st));
  const auto* base = static_cast<const char*>(proj);
  DecayedAttn d;
  d.dtype = dtype;
  d.q = base;
  d.k = base + static_cast<int64_t>(c.heads) * c.dim * esz();
  d.v = base + 2 * static_cast<int64_t>(c.heads) * c.dim * esz();
  d.ld = L.in_w; d.o = att; d.ld_o = L.att_w;
  d.state = L.state; d.decay = L.decay;
  d.batch = batch; d.len = n; d.heads = c.heads; d.dim = c.dim; d.vdim = c.vdim;
  d.first = len == 0;
  LM_TRY(decayed_attention(d, st));
  GatedRows g;
  g.dtype = dtype;
  g.in = g.out = att; g.ld_in = g.ld_out = L.att_w;
  g.gate = base + static_cast<int64_t>(L.gate_off) * esz(); g.ld_gate = L.in_w;
  g.rows = n_rows; g.cols = L.att_w; g.width = c.norm_width; g.w = L.mix_norm; g.eps = eps;
  return gated_rows(g, st);
}

int DerupelModel::pass(const int* ids, int n, const int* want, int n_want, float* logits, cudaStream_t st) {
  const int w = width;
  const int64_t n_rows = static_cast<int64_t>(batch) * n;
  LM_TRY(embed_rows(embed, ids, x, n_rows, w, vocab, embed_scale, st));
  LM_TRY(clear_counts(st));
  ResidualNorm rn = residual(n_rows);  // what the next residual kernel adds to the stream: the sublayer before it
  for (size_t l = 0; l < layers.size(); ++l) {
    const DerupelLayer& L = layers[l];
    LM_TRY(residual_norm(rn, st));
    LM_TRY(L.is_latent() ? mix_latent(L, n, st) : mix_decayed(L, n, st));
    LM_TRY(linear(att, L.att_w, L.o, y, w, n_rows, w, L.att_w, epilogue(EPI_NONE), true, st));
    rn.y = y;
    rn.slot = nullptr;
    rn.w_post = L.norm1;
    if (L.c.mlp == YTC_MLP_NONE) continue;
    LM_TRY(residual_norm(rn, st));
    rn.w_post = L.norm2;
    if (L.c.mlp == YTC_MLP_DENSE) {
      LM_TRY(linear(h, w, L.up, act, L.c.ff, n_rows, L.c.ff, w, epilogue(EPI_RELU2), false, st));
      LM_TRY(linear(act, L.c.ff, L.down, y, w, n_rows, w, L.c.ff, epilogue(EPI_NONE), true, st));
    } else {
      LM_TRY(moe_pass(L.moe, static_cast<int>(l), n_rows, rn, st));
    }
  }
  return logits_of(rn, want, n_want, logits, st);
}

int DerupelModel::step_latent(const DerupelLayer& L, cudaStream_t st) {
  const ytcuda_derupel_layer& c = L.c;
  LM_TRY(step_linear(step_input(nullptr), L.in, L.in_w, width, epilogue(EPI_NONE), sproj, nullptr, st));
  DecodeInput cqn;
  cqn.kind = DECODE_GATED;
  cqn.plain = sproj; cqn.w_pre = L.dq_norm; cqn.width = c.q_width; cqn.eps = eps;
  LM_TRY(step_linear(cqn, L.uq, L.q_w(), c.q_rank, epilogue(EPI_NONE), sq, nullptr, st));
  LatentAppend ap = append_of(L);
  ap.in = sproj; ap.pos = pos;
  LatentDecode d;
  d.dtype = dtype; d.io_dtype = YTC_F32;
  d.s = L.latent;
  d.q = sq; d.uk = L.uk; d.uv = L.uv; d.cache = L.cache; d.cap = max_tokens;
  d.pos = pos; d.max_keys = max_tokens; d.scale = c.scale;
  d.qa = sqa; d.part = spart; d.out = satt; d.ld_out = L.att_w;
  d.append = &ap;
  LM_TRY(latent_decode(d, st));
  DecodeInput gated;
  gated.kind = DECODE_GATED;
  gated.plain = satt; gated.gate = sproj + L.gate_off; gated.width = L.att_w; gated.eps = eps;
  return step_linear(gated, L.o, width, L.att_w, epilogue(EPI_NONE), sy, nullptr, st);
}

int DerupelModel::step_decayed(const DerupelLayer& L, cudaStream_t st) {
  const ytcuda_derupel_layer& c = L.c;
  LinearEpilogue silu = epilogue(EPI_SILU);
  silu.act_cols = L.gate_off;
  LM_TRY(step_linear(step_input(nullptr), L.in, L.in_w, width, silu, sproj, nullptr, st));
  DecayedAttn d;
  d.dtype = YTC_F32;
  d.q = sproj; d.k = sproj + c.heads * c.dim; d.v = sproj + 2 * c.heads * c.dim;
  d.ld = L.in_w; d.o = satt; d.ld_o = L.att_w;
  d.state = L.state; d.decay = L.decay; d.pos = pos;
  d.heads = c.heads; d.dim = c.dim; d.vdim = c.vdim;
  LM_TRY(decayed_attention(d, st));
  DecodeInput gated;
  gated.kind = DECODE_GATED;
  gated.plain = satt; gated.gate = sproj + L.gate_off; gated.w_pre = L.mix_norm; gated.width = c.norm_width; gated.eps = eps;
  return step_linear(gated, L.o, width, L.att_w, epilogue(EPI_NONE), sy, nullptr, st);
}

int DerupelModel::step_launches(cudaStream_t st) {
  const int w = width;
  for (const DerupelLayer& L : layers) {
    LM_TRY(L.is_latent() ? step_latent(L, st) : step_decayed(L, st));
    step_post = L.norm1;
    if (L.c.mlp == YTC_MLP_NONE) continue;
    if (L.c.mlp == YTC_MLP_DENSE) {
      LM_TRY(step_linear(step_input(nullptr), L.up, L.c.ff, w, epilogue(EPI_RELU2), sact, nullptr, st));
      LM_TRY(step_linear(step_plain(sact), L.down, w, L.c.ff, epilogue(EPI_NONE), sy, nullptr, st));
    } else {
      LM_TRY(step_moe(L.moe, nullptr, st));
    }
    step_post = L.norm2;
  }
  return step_linear(step_input(final_norm), head, vocab, w, epilogue(EPI_NONE), step_logits, pos, st);
}

static const char* bad_layer(const ytcuda_derupel_layer& c) {
  if (c.mixer != YTC_MIXER_DECAYED && c.mixer != YTC_MIXER_LATENT) return "unknown mixer";
  if (c.heads <= 0 || c.dim <= 0 || c.dim % 8 || c.vdim <= 0 || c.vdim % 8) return "head dims must be multiples of 8";
  if (c.mixer == YTC_MIXER_DECAYED) {
    if (c.dim > 512) return "heads of more than 512 dimensions";
    if (c.norm_width <= 0 || c.norm_width > c.heads * c.vdim) return "bad norm width";
  } else {
    if (c.rot < 0 || c.rot % 16 || c.rot_dims < 0 || c.rot_dims % 2 || c.rot_dims > c.rot || c.rot_dims > 256)
      return "rotated dimensions must be even, at most 256, stored in multiples of 16";
    if (c.head_ld < c.dim + c.rot || c.head_ld % 8 || c.head_ld > 256 || c.vdim > 256)
      return "heads of more than 256 dimensions";
    if (c.rank <= 0 || c.rank % 16 || c.rank > 1024 || c.q_rank <= 0 || c.q_rank % 8)
      return "latents must be multiples of 16 (queries: 8), at most 1024";
    if (c.q_width <= 0 || c.q_width > c.q_rank || c.c_width <= 0 || c.c_width > c.rank) return "bad norm width";
  }
  if (c.mlp < YTC_MLP_NONE || c.mlp > YTC_MLP_MOE) return "unknown feed-forward kind";
  if (c.mlp != YTC_MLP_NONE && (c.ff <= 0 || c.ff % 8)) return "the feed-forward width must be a multiple of 8";
  if (c.mlp == YTC_MLP_MOE) {
    if (c.experts <= 0 || c.experts > LM_MAX_ROUTES || c.top <= 0 || c.top > c.experts || c.top > LM_MAX_TOP)
      return "bad number of experts";
    if (c.shared_ff < 0 || c.shared_ff % 8) return "the shared expert's width must be a multiple of 8";
  }
  return nullptr;
}

}  // namespace ytk

using namespace ytk;

extern "C" {

void* ytcuda_derupel_create(const ytcuda_derupel_config* cfg, const ytcuda_derupel_layer* layers) {
  if (!cfg || !layers || cfg->layers <= 0) {
    set_last_error("ytcuda_derupel_create: no layers");
    return nullptr;
  }
  auto m = std::make_unique<DerupelModel>();
  m->width = cfg->width; m->norm_width = cfg->norm_width; m->vocab = cfg->vocab; m->batch = cfg->batch;
  m->max_tokens = cfg->max_tokens; m->chunk = std::min(cfg->chunk, cfg->max_tokens); m->dtype = cfg->dtype; m->eps = cfg->eps;
  m->embed_scale = cfg->embed_scale;
  if (!m->check_config("ytcuda_derupel_create")) return nullptr;
  for (int l = 0; l < cfg->layers; ++l) {
    DerupelLayer L;
    L.c = layers[l];
    const ytcuda_derupel_layer& c = L.c;
    if (const char* why = bad_layer(c)) {
      set_last_error("ytcuda_derupel_create: layer %d: %s", l, why);
      return nullptr;
    }
    L.att_w = c.heads * c.vdim;
    if (L.is_latent()) {
      LatentShape& s = L.latent;
      s.heads = c.heads; s.dim = c.dim; s.rot = c.rot; s.vdim = c.vdim; s.head_ld = c.head_ld; s.rank = c.rank;
      s.rot_dims = c.rot_dims;
      L.gate_off = c.q_rank + s.row();
    } else {
      L.gate_off = c.heads * (2 * c.dim + c.vdim);
    }
    L.in_w = L.gate_off + L.att_w;
    if (c.mlp == YTC_MLP_MOE) {
      L.moe.route = RouterSpec{c.experts, 0, c.top, 1, 1, ROUTE_SIGMOID};
      L.moe.ff = c.ff;
      L.moe.act = L.moe.shared_act = epilogue(EPI_CLAMP_PAIRS);
      L.moe.act.limit = c.limit;
      L.moe.shared_act.limit = c.shared_limit;
      L.moe.scale_input = true;
      L.moe.shared_ff = c.shared_ff;
    }
    m->layers.push_back(L);
  }
  bool ok = m->alloc_counts() == YTC_OK;
  for (DerupelLayer& L : m->layers) {
    if (L.is_latent())
      ok = ok && m->alloc(L.cache, static_cast<int64_t>(m->batch) * m->max_tokens * L.latent.row() * m->esz()) == YTC_OK;
    else
      ok = ok && m->alloc(L.state, static_cast<int64_t>(m->batch) * L.c.heads * L.c.dim * L.c.vdim * 4) == YTC_OK;
  }
  if (!ok) {
    set_last_error("ytcuda_derupel_create: device allocation failed");
    return nullptr;
  }
  return static_cast<LmModel*>(m.release());
}

int ytcuda_derupel_set_weight(void* handle, const char* name, int layer, const void* dptr) {
  auto* m = static_cast<DerupelModel*>(static_cast<LmModel*>(handle));
  YTC_REQUIRE(m && name && dptr, "ytcuda_derupel_set_weight: null argument");
  YTC_REQUIRE((reinterpret_cast<uint64_t>(dptr) & 15) == 0, "ytcuda_derupel_set_weight: weights must be 16-byte aligned");
  const std::string n(name);
  const auto* f = static_cast<const float*>(dptr);
  const auto* b = static_cast<const uint16_t*>(dptr);
  if (m->set_common_weight(n, dptr)) return YTC_OK;
  YTC_REQUIRE(layer >= 0 && layer < static_cast<int>(m->layers.size()), "ytcuda_derupel_set_weight: layer %d out of range",
              layer);
  DerupelLayer& L = m->layers[layer];
  const bool moe = L.c.mlp == YTC_MLP_MOE;
  if (n == "norm1") L.norm1 = f;
  else if (n == "norm2") L.norm2 = f;
  else if (n == "in") L.in = b;
  else if (n == "o") L.o = b;
  else if (n == "mix_norm") L.mix_norm = f;
  else if (n == "decay") L.decay = f;
  else if (n == "dq_norm") L.dq_norm = f;
  else if (n == "dkv_norm") L.dkv_norm = f;
  else if (n == "freq") L.latent.freq = f;
  else if (n == "uq") L.uq = b;
  else if (n == "uk") L.uk = b;
  else if (n == "uv") L.uv = b;
  else if (n == "expand") L.expand = b;
  else if (n == "up") (moe ? L.moe.up : L.up) = b;
  else if (n == "down") (moe ? L.moe.down : L.down) = b;
  else if (n == "router") L.moe.router = b;
  else if (n == "shared_up") L.moe.shared_up = b;
  else if (n == "shared_down") L.moe.shared_down = b;
  else {
    set_last_error("ytcuda_derupel_set_weight: unknown weight name '%s'", name);
    return YTC_INVALID_ARG;
  }
  return YTC_OK;
}

}  // extern "C"
