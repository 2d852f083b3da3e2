// The prepared model and the session: what runtime.cu (the session verbs and the uniform decoder's step) and
// layered.cu (the step of decoders described layer by layer) share.
#pragma once

#include <algorithm>
#include <map>
#include <memory>
#include <mutex>
#include <string>
#include <vector>

#include "abi_util.cuh"
#include "kernels.cuh"
#include "smallm_gemm.cuh"

namespace ei {

constexpr size_t kAlign = 256;
constexpr int kMaxRows = 16;

inline size_t aligned(size_t bytes) { return (bytes + kAlign - 1) & ~(kAlign - 1); }

struct PreparedLinear {
  bool quantized = false;
  int in = 0, out = 0;
  const int32_t* qweight = nullptr;
  const bf16* scales = nullptr;
  const int32_t* zeros = nullptr;
  int padded_groups = 0, zero_stride = 0, group_size = 0;
  const bf16* dense = nullptr;  // [out, in]
  const bf16* bias = nullptr;
  int activation = kActNone;    // of a stored result
  int glu = kGluSilu;           // a gate|up pair: which gated unit its epilogue applies
  float glu_limit = 0.0f;
  size_t bytes = 0;  // weight bytes one call streams
};

constexpr size_t kPromptSegment = 2048;  // rows of a long prompt that go through the layers together

struct LayeredModel;
struct LayeredSession;

}  // namespace ei

struct ei_model {
  ei_model_config config{};
  int device = 0;
  unsigned char* arena = nullptr;
  size_t arena_bytes = 0;
  const ei::bf16* embedding = nullptr;
  const ei::bf16* output_norm = nullptr;
  ei::PreparedLinear lm_head;
  struct Layer {
    ei::PreparedLinear qkv, o, gate_up, down;
    const ei::bf16 *attention_norm = nullptr, *ffn_norm = nullptr, *q_norm = nullptr, *k_norm = nullptr;
  };
  std::vector<Layer> layers;
  float* rope_table = nullptr;
  size_t weight_bytes = 0;
  int multiprocessors = 1;  // queried at creation
  size_t smem_limit = 227 * 1024;
  // Activations of a prompt segment (up to kPromptSegment rows through every projection at once): one set per
  // model, created by the first long prompt and lent, under the mutex, to one prefill at a time.
  struct PromptWorkspace {
    std::mutex mutex;
    unsigned char* arena = nullptr;
    size_t rows = 0;
    ei::bf16 *residual = nullptr, *normed = nullptr, *qkv = nullptr, *attention = nullptr, *gate_up = nullptr,
         *act = nullptr, *projection = nullptr;
    float* partial = nullptr;         // FP32 sums of the o / down projections: [K slices][rows][hidden]
    size_t partial_bytes = 0;
    uint32_t *tokens = nullptr, *step_tokens = nullptr;
    uint32_t* host_tokens = nullptr;  // pinned
  } prompt;
  std::shared_ptr<ei::LayeredModel> layered;  // set for decoders described layer by layer (layered.cu)
  bool prompt_ready = false;  // every projection of every layer has a shape the prompt GEMM takes
};

struct ei_session {
  ei_model* model = nullptr;
  size_t capacity = 0;
  bool use_graph = false;
  cudaStream_t stream = nullptr;
  unsigned char* arena = nullptr;
  // workspace
  ei::bf16 *residual = nullptr, *normed = nullptr, *qkv = nullptr, *attention = nullptr, *act = nullptr,
       *gate_up = nullptr, *projection = nullptr, *logits = nullptr;
  float* partial = nullptr;
  float* attention_scratch = nullptr;
  float* best_value = nullptr;
  int* best_index = nullptr;
  uint32_t *tokens = nullptr, *step_tokens = nullptr, *targets = nullptr;
  int32_t* gather_index = nullptr;      // places of the rows whose logits are asked for
  ei::Control* control = nullptr;
  ei::DraftSource* draft_source = nullptr;
  ei::DraftSource draft_host{nullptr, 0, 0};
  ei::TokenSink* token_sink = nullptr;  // device; all zero unless a speculative decoder owns the session
  ei::bf16 *k_cache = nullptr, *v_cache = nullptr;
  // pinned host staging
  uint32_t* host_tokens = nullptr;
  ei::Control* host_control = nullptr;
  // plans
  int attention_chunk = 64, attention_splits = 1;
  std::shared_ptr<ei::LayeredSession> layered;  // caches, recurrent state and buffers of a layered decoder
  // state
  size_t context = 0;
  size_t bound = 0;  // upper bound of the context length after every step enqueued so far (full acceptance)
  bool history_ready = false, poisoned = false;
  int inject_launch = 0, inject_completion = 0;
  uint32_t inject_attention_polls = 0;  // the same hook for the next attention launch (its K / V tile copies)
  uint32_t inject_wait_polls = 0;  // test hook: the next weight-streaming GEMM gets this poll limit and a copy
                                   // expectation it cannot meet, so that its bounded waits run out
  size_t launches = 0, launches_per_step[ei::kMaxRows + 1] = {};
  size_t prefill_target_row = 0;  // where in `targets` the last prefill left the greedy token of its last row
  // graphs: [kind][rows]; kind 0 verify (host tokens), 1 verify (device drafts), 2 decode (commit all)
  cudaGraphExec_t graphs[3][ei::kMaxRows + 1] = {};
};

namespace ei {

enum StepKind { kVerifyHost = 0, kVerifyDevice = 1, kCommitAllWithHead = 2, kCommitAllNoHead = 3 };

// Counts a launch of the session (and fails it when the test hook is armed).
void tick(ei_session& s);
// One projection of at most 16 rows by the weight-streaming kernels (s.partial / s.best_* are its outputs where the
// epilogue says so), and whether a plan exists for it. x_stride 0: rows of w.in inputs side by side.
void run_linear(ei_session& s, const PreparedLinear& w, const bf16* x, int rows, int epilogue, bf16* out,
                int out_stride, bool pdl, int* ksplit_out = nullptr, int x_stride = 0);
bool has_plan(const ei_session& s, const PreparedLinear& w, int rows, int epilogue);
// One projection of a prompt segment on the tensor cores; ksplit == 0: BF16 output with bias, otherwise FP32 partial
// sums of `ksplit` K slices in `partial` (null: the model's prompt workspace).
bool prompt_linear_ok(const PreparedLinear& w);
void run_prompt_linear(ei_session& s, const PreparedLinear& w, const bf16* x, int rows, bf16* out, bool pdl,
                       int ksplit = 0, int x_stride = 0, float* partial = nullptr);
void run_prompt_linear_store(ei_session& s, const PreparedLinear& w, const bf16* x, int rows, bf16* out, bool pdl,
                             int x_stride = 0);
// Commits all rows of a step. `folded`: the step's kernels already carried their recurrent state past these rows (a
// prompt segment); otherwise the rows stay pending behind Control::state_base.
void enqueue_commit(ei_session& s, int rows, bool folded);

}  // namespace ei
