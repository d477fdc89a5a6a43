// Duzozen decoder-only language model: per layer a norm before and after each sublayer, sliding-window attention with
// capped scores and no rotation, values mixed with the first mixing layer's, and a dense or mixture-of-experts
// feed-forward. This file is the model's own host side: weights, K/V rings, buffers and the order of launches; passes,
// decode graph and experts are LmModel's (lm_model.cuh), the mechanisms are in lm_ops.cuh (window_attention, append_kv,
// residual_norm, linear_tc / linear_f32, moe_*, decode_*). A pass has at most `chunk` tokens per sequence, so that a
// window's ring holds window - 1 + chunk positions however long the sequence is.
#include "lm_model.cuh"

namespace ytk {

struct DuzozenLayer {
  ytcuda_duzozen_layer c{};
  const float *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr, *vmix = nullptr;
  const uint16_t *qkv = nullptr, *o = nullptr, *up = nullptr, *down = nullptr;
  MoeLayer moe;
  int qkv_w = 0, att_w = 0, mix = VMIX_NONE;
  int ring = 0;
  void *k = nullptr, *v = nullptr;  // [batch][kv_heads][ring][dim / vdim]
};

struct DuzozenModel : LmModel {
  std::vector<DuzozenLayer> layers;
  void *qkv = nullptr, *att = nullptr, *act = nullptr, *v_first = nullptr;  // of a pass
  float *sqkv = nullptr, *satt = nullptr, *sv_first = nullptr;              // of a decode step

  int64_t qkv_width() const {
    int64_t n = 0;
    for (const DuzozenLayer& L : layers) n = std::max<int64_t>(n, L.qkv_w);
    return n;
  }
  int64_t att_width() const {
    int64_t n = 0;
    for (const DuzozenLayer& L : layers) n = std::max<int64_t>(n, L.att_w);
    return n;
  }
  int64_t v_first_width() const {
    int64_t n = 0;
    for (const DuzozenLayer& L : layers)
      if (L.mix != VMIX_NONE) n = std::max<int64_t>(n, static_cast<int64_t>(L.c.kv_heads) * L.c.vdim);
    return n;
  }
  int step_act_floats() const override {  // (of the dense layers)
    int n = 0;
    for (const DuzozenLayer& L : layers) n = std::max(n, L.c.mlp == YTC_MLP_DENSE ? L.c.ff : 0);
    return n;
  }
  std::vector<const MoeLayer*> moe_layers() const override {
    std::vector<const MoeLayer*> v;
    for (const DuzozenLayer& L : layers) v.push_back(L.c.mlp == YTC_MLP_MOE ? &L.moe : nullptr);
    return v;
  }
  int alloc_pass(int64_t r) override {
    const int64_t e = esz();
    LM_TRY(pass_alloc(qkv, r * qkv_width() * e));
    LM_TRY(pass_alloc(att, r * att_width() * e));
    LM_TRY(pass_alloc(act, r * step_act_floats() * e));
    return pass_alloc(v_first, r * v_first_width() * e);
  }
  int alloc_step() override {
    LM_TRY(alloc(sqkv, qkv_width() * 4));
    LM_TRY(alloc(satt, att_width() * 4));
    return alloc(sv_first, std::max<int64_t>(1, v_first_width()) * 4);
  }
  bool weights_set() const override {
    for (const DuzozenLayer& L : layers) {
      bool ok = L.norm1 && L.norm1b && L.qkv && L.o && (L.mix != VMIX_MIX || L.vmix);
      if (L.c.mlp != YTC_MLP_NONE) ok = ok && L.norm2 && L.norm2b;
      if (L.c.mlp == YTC_MLP_DENSE) ok = ok && L.up && L.down;
      if (L.c.mlp == YTC_MLP_MOE)
        ok = ok && L.moe.router && L.moe.correction && (L.c.experts == 0 || (L.moe.up && L.moe.down));
      if (!ok) return false;
    }
    return true;
  }
  int pass(const int* ids, int n, const int* want, int n_want, float* logits, cudaStream_t st) override;
  int step_launches(cudaStream_t st) override;
};

int DuzozenModel::pass(const int* ids, int n, const int* want, int n_want, float* logits, cudaStream_t st) {
  const int B = batch, w = width;
  const int64_t n_rows = static_cast<int64_t>(B) * n;
  LM_TRY(embed_rows(embed, ids, x, n_rows, w, vocab, embed_scale, st));
  LM_TRY(clear_counts(st));
  ResidualNorm rn = residual(n_rows);  // what the next residual kernel adds to the stream: the sublayer before it
  for (size_t l = 0; l < layers.size(); ++l) {
    const DuzozenLayer& L = layers[l];
    const ytcuda_duzozen_layer& c = L.c;
    rn.w_pre = L.norm1;
    LM_TRY(residual_norm(rn, st));
    LM_TRY(linear(h, w, L.qkv, qkv, L.qkv_w, n_rows, L.qkv_w, w, epilogue(EPI_NONE), false, st));
    AppendKv ap;
    ap.dtype = dtype;
    ap.qkv = qkv; ap.ld = L.qkv_w;
    ap.k_off = c.heads * c.dim; ap.v_off = (c.heads + c.kv_heads) * c.dim;
    ap.k = L.k; ap.v = L.v;
    ap.v_first = v_first; ap.lambda = L.vmix; ap.mix = L.mix;
    ap.batch = B; ap.len = n; ap.kv_heads = c.kv_heads; ap.dim = c.dim; ap.vdim = c.vdim; ap.ring = L.ring;
    ap.pos0 = len;
    LM_TRY(append_kv(ap, st));
    WindowAttn at;
    at.dtype = dtype;
    at.q = qkv; at.k = L.k; at.v = L.v; at.o = att;
    at.batch = B; at.kv_heads = c.kv_heads; at.groups = c.heads / c.kv_heads; at.q_len = n;
    at.head_dim = c.dim; at.value_dim = c.vdim;
    at.q_st[0] = static_cast<int64_t>(n) * L.qkv_w; at.q_st[1] = c.dim; at.q_st[2] = L.qkv_w;
    at.k_st[0] = static_cast<int64_t>(c.kv_heads) * L.ring * c.dim; at.k_st[1] = static_cast<int64_t>(L.ring) * c.dim; at.k_st[2] = c.dim;
    at.v_st[0] = static_cast<int64_t>(c.kv_heads) * L.ring * c.vdim; at.v_st[1] = static_cast<int64_t>(L.ring) * c.vdim; at.v_st[2] = c.vdim;
    at.o_st[0] = static_cast<int64_t>(n) * L.att_w; at.o_st[1] = c.vdim; at.o_st[2] = L.att_w;
    at.pos0 = len; at.window = c.window; at.ring = L.ring;
    at.scale = c.scale; at.softcap = c.softcap;
    LM_TRY(window_attention(at, st));
    LM_TRY(linear(att, L.att_w, L.o, y, w, n_rows, w, L.att_w, epilogue(EPI_NONE), true, st));
    rn.y = y;
    rn.slot = nullptr;
    rn.w_post = L.norm1b;
    if (c.mlp == YTC_MLP_NONE) continue;
    rn.w_pre = L.norm2;
    LM_TRY(residual_norm(rn, st));
    rn.w_post = L.norm2b;
    if (c.mlp == YTC_MLP_DENSE) {
      LM_TRY(linear(h, w, L.up, act, c.ff, n_rows, c.ff, w, epilogue(EPI_GELU_ERF), false, st));
      LM_TRY(linear(act, c.ff, L.down, y, w, n_rows, w, c.ff, epilogue(EPI_NONE), true, st));
    } else {
      LM_TRY(moe_pass(L.moe, static_cast<int>(l), n_rows, rn, st));
    }
  }
  return logits_of(rn, want, n_want, logits, st);
}

int DuzozenModel::step_launches(cudaStream_t st) {
  const int w = width;
  for (const DuzozenLayer& L : layers) {
    const ytcuda_duzozen_layer& c = L.c;
    LM_TRY(step_linear(step_input(L.norm1), L.qkv, L.qkv_w, w, epilogue(EPI_NONE), sqkv, nullptr, st));
    DecodeAttn at;
    at.dtype = dtype;
    at.qkv = sqkv; at.k = L.k; at.v = L.v; at.v_first = sv_first; at.lambda = L.vmix; at.mix = L.mix;
    at.out = satt; at.pos = pos;
    at.kv_heads = c.kv_heads; at.groups = c.heads / c.kv_heads; at.dim = c.dim; at.vdim = c.vdim;
    at.ring = L.ring; at.window = c.window;
    at.max_keys = c.window > 0 ? std::min<int64_t>(c.window, max_tokens) : max_tokens;
    at.scale = c.scale; at.softcap = c.softcap;
    LM_TRY(decode_attention(at, st));
    LM_TRY(step_linear(step_plain(satt), L.o, w, L.att_w, epilogue(EPI_NONE), sy, nullptr, st));
    step_post = L.norm1b;
    if (c.mlp == YTC_MLP_NONE) continue;
    if (c.mlp == YTC_MLP_DENSE) {
      LM_TRY(step_linear(step_input(L.norm2), L.up, c.ff, w, epilogue(EPI_GELU_ERF), sact, nullptr, st));
      LM_TRY(step_linear(step_plain(sact), L.down, w, c.ff, epilogue(EPI_NONE), sy, nullptr, st));
    } else {
      LM_TRY(step_moe(L.moe, L.norm2, st));
    }
    step_post = L.norm2b;
  }
  return step_linear(step_input(final_norm), head, vocab, w, epilogue(EPI_NONE), step_logits, pos, st);
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
  if (!cfg || !layers || cfg->layers <= 0) {
    set_last_error("ytcuda_duzozen_create: no layers");
    return nullptr;
  }
  auto m = std::make_unique<DuzozenModel>();
  m->width = cfg->width; m->norm_width = cfg->norm_width; m->vocab = cfg->vocab; m->batch = cfg->batch;
  m->max_tokens = cfg->max_tokens; m->chunk = std::min(cfg->chunk, cfg->max_tokens); m->dtype = cfg->dtype; m->eps = cfg->eps;
  if (!m->check_config("ytcuda_duzozen_create")) return nullptr;
  bool first_seen = false;
  int vf = 0;
  for (int l = 0; l < cfg->layers; ++l) {
    DuzozenLayer L;
    L.c = layers[l];
    std::string why;
    if (bad_layer(L.c, &why)) {
      set_last_error("ytcuda_duzozen_create: layer %d: %s", l, why.c_str());
      return nullptr;
    }
    L.qkv_w = (L.c.heads + L.c.kv_heads) * L.c.dim + L.c.kv_heads * L.c.vdim;
    L.att_w = L.c.heads * L.c.vdim;
    if (L.c.v_mix) {
      const int mine = L.c.kv_heads * L.c.vdim;
      if (first_seen && mine != vf) {
        set_last_error("ytcuda_duzozen_create: layer %d mixes values of another size than the first mixing layer's", l);
        return nullptr;
      }
      L.mix = first_seen ? VMIX_MIX : VMIX_FIRST;
      first_seen = true;
      vf = mine;
    }
    if (L.c.mlp == YTC_MLP_MOE) {
      L.moe.route = RouterSpec{L.c.experts, L.c.identity, L.c.top, L.c.groups, L.c.keep};
      L.moe.ff = L.c.ff;
      L.moe.act = epilogue(EPI_SWIGLU_PAIRS);
    }
    // Rings are whole tiles of 128 positions. A pass of `chunk` tokens needs the window before its first token and
    // itself, wherever these fall between tile borders.
    auto tile = [](int64_t n) { return (n + 127) / 128 * 128; };
    int64_t ring = tile(m->max_tokens);
    if (L.c.window > 0) ring = std::min(ring, tile(static_cast<int64_t>(L.c.window) - 1 + m->chunk) + 128);
    L.ring = static_cast<int>(ring);
    m->layers.push_back(L);
  }
  bool ok = m->alloc_counts() == YTC_OK;
  for (DuzozenLayer& L : m->layers) {
    const size_t kb = static_cast<size_t>(cfg->batch) * L.c.kv_heads * L.ring * L.c.dim * m->esz();
    const size_t vb = static_cast<size_t>(cfg->batch) * L.c.kv_heads * L.ring * L.c.vdim * m->esz();
    ok = ok && m->alloc(L.k, kb) == YTC_OK && m->alloc(L.v, vb) == YTC_OK && cudaMemset(L.k, 0, kb) == cudaSuccess &&
         cudaMemset(L.v, 0, vb) == cudaSuccess;
  }
  if (!ok) {
    set_last_error("ytcuda_duzozen_create: device allocation failed");
    return nullptr;
  }
  return static_cast<LmModel*>(m.release());
}

int ytcuda_duzozen_set_weight(void* handle, const char* name, int layer, const void* dptr) {
  auto* m = static_cast<DuzozenModel*>(static_cast<LmModel*>(handle));
  YTC_REQUIRE(m && name && dptr, "ytcuda_duzozen_set_weight: null argument");
  YTC_REQUIRE((reinterpret_cast<uint64_t>(dptr) & 15) == 0, "ytcuda_duzozen_set_weight: weights must be 16-byte aligned");
  const std::string n(name);
  const auto* f = static_cast<const float*>(dptr);
  const auto* b = static_cast<const uint16_t*>(dptr);
  if (m->set_common_weight(n, dptr)) return YTC_OK;
  YTC_REQUIRE(layer >= 0 && layer < static_cast<int>(m->layers.size()), "ytcuda_duzozen_set_weight: layer %d out of range",
              layer);
  DuzozenLayer& L = m->layers[layer];
  const bool moe = L.c.mlp == YTC_MLP_MOE;
  if (n == "norm1") L.norm1 = f;
  else if (n == "norm1b") L.norm1b = f;
  else if (n == "norm2") L.norm2 = f;
  else if (n == "norm2b") L.norm2b = f;
  else if (n == "vmix") L.vmix = f;
  else if (n == "correction") L.moe.correction = f;
  else if (n == "qkv") L.qkv = b;
  else if (n == "o") L.o = b;
  else if (n == "up") (moe ? L.moe.up : L.up) = b;
  else if (n == "down") (moe ? L.moe.down : L.down) = b;
  else if (n == "router") L.moe.router = b;
  else {
    set_last_error("ytcuda_duzozen_set_weight: unknown weight name '%s'", name);
    return YTC_INVALID_ARG;
  }
  return YTC_OK;
}

}  // extern "C"
