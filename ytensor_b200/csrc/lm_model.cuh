// What the language models of the library share on the host: device buffers, a forward call cut into passes, the CUDA
// graph of a decode step, linear layers in the model's number format and the mixture-of-experts feed-forward. A model
// derives from LmModel and supplies its layers (csrc/duzozen.cu, csrc/derupel.cu).
#pragma once
#include <algorithm>
#include <memory>
#include <string>
#include <vector>

#include "lm_ops.cuh"

namespace ytk {

#define LM_TRY(expr)                 \
  do {                               \
    const int _s = (expr);           \
    if (_s != YTC_OK) return _s;     \
  } while (0)

// Feed-forward with experts; what one expert computes is `act` (EPI_SWIGLU_PAIRS / EPI_CLAMP_PAIRS) between its gate /
// up rows and its down rows. The shared expert runs for every token and is added.
struct MoeLayer {
  RouterSpec route;
  const uint16_t* router = nullptr;   // [experts + identity][width]
  const float* correction = nullptr;  // [experts + identity] or null
  const uint16_t *up = nullptr, *down = nullptr;  // [experts][2 ff][width] gate_j, up_j alternating; [experts][width][ff]
  int ff = 0;
  LinearEpilogue act;
  bool scale_input = false;  // the route's weight multiplies the expert's input instead of its output
  const uint16_t *shared_up = nullptr, *shared_down = nullptr;
  int shared_ff = 0;         // 0: no shared expert
  LinearEpilogue shared_act;
  int routes() const { return route.experts + route.identity; }
};

struct LmModel {
  int width = 0, norm_width = 0, vocab = 0, batch = 1, max_tokens = 0, chunk = 0, dtype = YTC_F32;
  float eps = 0.f, embed_scale = 1.f;
  const uint16_t *embed = nullptr, *head = nullptr;
  const float* final_norm = nullptr;
  int64_t len = 0;        // tokens in every sequence
  int decode_path = 0;    // 0: the graph of fused kernels for one token of one sequence, 1: the operator path always
  std::vector<void*> owned;
  // buffers of a pass of `rows` rows; alloc_pass() adds the model's
  int64_t rows = 0;
  std::vector<void*> pass_owned;
  float *x = nullptr, *y = nullptr, *logit = nullptr, *weight = nullptr;
  void *h = nullptr, *hf = nullptr, *shared_act = nullptr, *grouped = nullptr, *expert_act = nullptr, *expert_out = nullptr;
  int *ids = nullptr, *want = nullptr, *choice = nullptr, *rank = nullptr, *slot = nullptr, *tile_group = nullptr,
      *count = nullptr;
  // decode step
  bool step_ready = false;
  int64_t dev_pos = -1;   // what the position word on the device holds
  int *pos = nullptr, *step_id = nullptr, *step_choice = nullptr;
  float *sx[2] = {}, *sy = nullptr, *sact = nullptr, *sh = nullptr, *step_weight = nullptr, *step_logits = nullptr;
  cudaStream_t cap_stream = nullptr;
  cudaGraphExec_t step = nullptr;
  int step_kernels = 0;

  virtual ~LmModel();
  bool bf16() const { return dtype == YTC_BF16; }
  int esz() const { return bf16() ? 2 : 4; }
  // What ytcuda_*_create checks of every model; false with the error text set.
  bool check_config(const char* name) const;

  // ---- what a model supplies
  virtual std::vector<const MoeLayer*> moe_layers() const = 0;  // (null where a layer has none)
  virtual int step_act_floats() const = 0;    // widest feed-forward activation of a decode step
  virtual int alloc_pass(int64_t rows) = 0;   // the model's own pass buffers (pass_alloc)
  virtual int alloc_step() = 0;               // the model's own decode buffers (alloc)
  virtual int pass(const int* ids, int n, const int* want, int n_want, float* logits, cudaStream_t st) = 0;
  virtual int step_launches(cudaStream_t st) = 0;
  virtual bool weights_set() const = 0;
  virtual int clear_state() { return YTC_OK; }  // recurrent state, at the start of a sequence

  // ---- shared
  template <typename P>
  int alloc(P*& p, int64_t bytes) { return alloc_in(owned, reinterpret_cast<void**>(&p), bytes); }
  template <typename P>
  int pass_alloc(P*& p, int64_t bytes) { return alloc_in(pass_owned, reinterpret_cast<void**>(&p), bytes); }
  int alloc_counts();  // once, when the layers are known
  int ensure_pass(int64_t rows);
  // y = epilogue(x . W^T): activations in the model's type, y in it too (to_f32: fp32).
  int linear(const void* x, int64_t ldx, const uint16_t* w, void* y, int64_t ldy, int64_t rows, int n, int k,
             LinearEpilogue ex, bool to_f32, cudaStream_t st) const;
  ResidualNorm residual(int64_t rows) const;  // over x, into h
  // Experts of h (and, scale_input, of the fp32 rows x): fills rn's slots, weights and, with a shared expert, y.
  int moe_pass(const MoeLayer& m, int layer, int64_t rows, ResidualNorm& rn, cudaStream_t st);
  int count_words() const;
  int clear_counts(cudaStream_t st);  // at the start of a pass
  // The wanted rows' last residual sum, final norm and logits.
  int logits_of(ResidualNorm rn, const int* want, int n_want, float* logits, cudaStream_t st);

  // ---- decode step: the input of a kernel is the residual row after the sublayer whose output is in sy
  int step_cur = 0;                   // sx[step_cur] holds the residual row
  const float* step_post = nullptr;   // norm behind that sublayer (null: the embedding comes first)
  void step_begin() { step_cur = 0; step_post = nullptr; }
  DecodeInput step_input(const float* w_pre);
  static DecodeInput step_plain(const float* v);
  int step_linear(const DecodeInput& in, const uint16_t* w, int n, int k, const LinearEpilogue& ex, float* out, int* advance,
                  cudaStream_t st) const;
  int step_moe(const MoeLayer& m, const float* w_pre, cudaStream_t st);

  void drop_step();
  int forward(const int32_t* ids, int len, const int32_t* want, int n_want, float* logits, cudaStream_t st);
  int reset();
  bool set_common_weight(const std::string& name, const void* p);

 private:
  int alloc_in(std::vector<void*>& list, void** p, int64_t bytes);
  int ensure_step();
  int build_step();
  int run_step(const int* id, bool want, float* logits, cudaStream_t st);
};

inline LinearEpilogue epilogue(int epi) {
  LinearEpilogue e;
  e.epi = epi;
  return e;
}

// The switch of the chained launches for the duration of a call (launch_overlapped, ytc_common.cuh).
struct OverlapGuard {
  OverlapGuard() { overlap_scope() = true; }
  ~OverlapGuard() { overlap_scope() = false; }
};

}  // namespace ytk
