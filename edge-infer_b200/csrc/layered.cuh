// Decoders described layer by layer: the operations their layers are made of, and the model and session parts that
// hold their weights, caches and recurrent state.
//
// Head sizes and widths are free. Every head is stored with its size rounded up to a multiple of 16 and every
// projection input to a multiple of 64, the padding zero in the weights, so that all shapes go through the same GEMMs,
// copies and MMA tiles; the true sizes enter only where a mean is taken.
//
// Activations are BF16 or, for a model that runs in true 32-bit, FP32: the kernels are templates over the element
// type. The residual stream, norms, angles, scores, softmax weights, gates and recurrent state are FP32 in both.
#pragma once

#include "session.cuh"

namespace ei {

constexpr int kPendingRows = 16;     // rows a step may leave pending behind the recurrent state
constexpr int kRingRows = 32;        // ring of a recurrence's inputs: pending rows and the rows of the step
constexpr int kMinGruStretch = 32;   // rows of a prompt stretch of the gated recurrence
constexpr int kLightningChunk = 128; // tokens of a prompt chunk of the decayed linear attention
constexpr int kMaxHeadDim = 512;
constexpr int kMaxLatent = 1024;     // values of the latent of latent attention

// tanh(alpha * x) * weight + bias; vectors padded with zeros to the row stride.
struct DynamicTanh {
  const bf16* weight = nullptr;
  const bf16* bias = nullptr;
  float alpha = 0.0f;
};

// What is added to the residual stream ahead of a layer: the embedding output of the row's token and / or a vector.
struct Injection {
  const uint32_t* tokens = nullptr;  // [rows]; with `table` set, table[token] is added
  const bf16* table = nullptr;       // [vocab, stride of the residual]
  const bf16* vector = nullptr;
  int vocab = 0;
};

// x = embedding (+ injected vector); normed = norm(x). One block per row.
struct LayeredEmbedParams {
  EmbedParams token;        // token selection (its table, norm and output fields are not used)
  const bf16* table;        // [vocab, residual_stride]
  const bf16* vector;       // added to the stream ahead of the first layer, or null
  DynamicTanh norm;
  float* residual;          // [rows, residual_stride]
  int residual_stride;
  void* normed;             // [rows, normed_stride]
  int normed_stride;
};
template <typename T>
void launch_layered_embed(const LayeredEmbedParams& p, cudaStream_t stream, bool pdl);

// The end of a sublayer and the start of the next: x += after(sum of partials); tap = x; x += injection;
// normed = before(x).
struct SublayerJoinParams {
  const float* partial;     // [ksplit, rows, residual_stride]
  int ksplit, rows;
  DynamicTanh after, before;
  float* residual;
  int residual_stride;
  float* tap;               // optional copy of the stream before the injection: [rows, tap_width]
  int tap_width;
  Injection inject;
  void* normed;
  int normed_stride;
};
template <typename T>
void launch_sublayer_join(const SublayerJoinParams& p, cudaStream_t stream, bool pdl);

// ---- blocks whose mixer and feed-forward read the same stream (parallel_block.cu) ----
// A row of a table picked by a token and the one before it, added to the token's embedding: row
// (previous * mul_prev + token * mul_cur) mod buckets, row `buckets` for a sequence's first token.
struct PairTable {
  const bf16* table = nullptr;       // [buckets + 1, stride]; null: none
  int stride = 0;
  unsigned long long buckets = 0, mul_prev = 0, mul_cur = 0;
  uint32_t* history = nullptr;       // [capacity]: the token of every position
};
// One or two layer norms of the same row: (x - mean) / sqrt(variance + eps) * weight over `width` values.
struct RowNorms {
  const bf16 *first = nullptr, *second = nullptr;  // weights, zero beyond the width; second may be null
  void *normed_first = nullptr, *normed_second = nullptr;
  int width = 0, stride = 0;         // stride of the normed rows
  float eps = 0.0f;
};
struct ParallelEmbedParams {
  EmbedParams token;        // token selection (its table, norm and output fields are not used)
  const bf16* table;        // [vocab, table_stride]
  int table_stride;
  PairTable pairs;
  float* residual;          // [rows, residual_stride]
  int residual_stride;
  RowNorms norms;
};
template <typename T>
void launch_parallel_embed(const ParallelEmbedParams& p, cudaStream_t stream, bool pdl);
// x += mixed_scale * sum(mixed) + fed_scale * sum(fed); tap = x; normed rows of x. One block per row.
struct ParallelJoinParams {
  const float *mixed, *fed;          // [ksplit, rows, residual_stride]; fed may be null
  int mixed_ksplit, fed_ksplit, rows;
  const bf16 *mixed_scale, *fed_scale;
  float* residual;
  int residual_stride;
  float* tap;                        // optional copy of the stream: [rows, tap_width]
  int tap_width;
  RowNorms norms;
};
template <typename T>
void launch_parallel_join(const ParallelJoinParams& p, cudaStream_t stream, bool pdl);

// Per (row, head): rotation of q and k, value norm, KV append; SiLU of the linear attention's q, k, v, whose k and v
// are also recorded in the ring when the step leaves its rows pending. In place in the fused projection output.
struct MixerPrepareParams {
  void* fused;              // [rows, stride]: q | k | v | linear q | k | v | gate
  int rows, stride;
  int heads, kv_heads, dim, vdim, dim_pad, vdim_pad, rot_dims;
  float eps;
  const float2* rotation;   // [capacity][rot_dims / 2] (cos, sin)
  const Control* control;
  int capacity;
  void *k_cache, *v_cache;  // [capacity, kv_heads * dim_pad], [capacity, kv_heads * vdim_pad]
  int lin_heads, lin_dim_pad, lin_vdim_pad;
  void *ring_k, *ring_v;    // [kRingRows, lin_heads * pad] or null
};
template <typename T>
void launch_mixer_prepare(const MixerPrepareParams& p, cudaStream_t stream, bool pdl);

// ---- softmax attention with free head sizes, scale and per-head sink (sized_attention.cu) ----
struct SizedAttentionParams {
  const void* q;            // row r, head h at q + r * q_stride + h * dim_pad
  int q_stride;
  const void *k, *v;        // token t, KV head g at k + t * k_stride + g * dim_pad, v + t * v_stride + g * vdim_pad
  int k_stride, v_stride;
  int rows, heads, kv_heads, dim_pad, vdim_pad;
  const void* shared;       // the last shared_pad values of every head's key, token t at shared + t * shared_stride
  int shared_stride, shared_pad;
  int tokens;               // rows of k and v (0: the capacity in whole tiles)
  bool fresh;               // k and v come from the preceding kernels, earlier tokens too
  const void* gate;         // finished output times sigmoid of row r, head h at gate + r * gate_stride + h * vdim_pad; or null
  int gate_stride;
  float scale, out_scale;   // out_scale multiplies the finished output
  const float* sink;        // [heads]: exp(sink) joins the denominator; or null
  const int32_t* device_offset;
  int capacity;
  int chunk, max_splits;    // step form
  float* scratch;           // [max_splits][rows * heads][vdim_pad + 4]
  void* out;                // row r, head h at out + r * out_stride + h * vdim_pad
  int out_stride;
  CUtensorMap k_map, v_map, shared_map;  // filled by the launch functions
  int k_shift, v_shift;     // log2 of the 16-byte pieces in one row of a staged box
  int* status;
  uint32_t wait_limit, fault_tx;
};
// Head sizes the tiled kernels take (the others use launch_plain_attention).
bool sized_attention_ok(int dim_pad, int vdim_pad);
size_t sized_attention_scratch_bytes(size_t rows, size_t heads, size_t vdim_pad, size_t capacity);
// Split form for at most 16 rows; leaves partials for launch_mixer_finish.
void launch_sized_attention_step(const SizedAttentionParams& p, cudaStream_t stream, bool pdl);
// Any number of rows, finished output.
void launch_sized_attention_prompt(const SizedAttentionParams& p, cudaStream_t stream, bool pdl);
// One block per (row, head), value sizes up to kMaxLatent, FP32 or BF16 operands, finished output.
template <typename T>
void launch_plain_attention(const SizedAttentionParams& p, cudaStream_t stream, bool pdl);

// ---- decayed linear attention (lightning.cu) ----
// One decay per token and head instead of one per head, for prompts of state-space layers: the row's step
// t = softplus(step + bias) scales what it writes, and the state decays by exp(-rate t).
struct TokenDecay {
  const bf16* step;         // row r, head h at step + r * step_stride + h; null: decays are LightningParams::powers
  int step_stride;
  const float *bias, *rate;
  const float* skip;        // [heads]: skip * v is added to the output; or null
  int key_heads;            // head h reads q and k of head h / (heads / key_heads)
  const float *ring_k, *ring_g, *ring_u;  // pending rows (outer_state.cu)
  float* totals;            // [chunks][heads]: logarithm of a chunk's decay
};
struct LightningParams {
  const void *q, *k, *v;    // row r at + r * stride, heads side by side
  int stride, rows, heads, dim_pad, vdim_pad;
  const void *ring_k, *ring_v;  // [kRingRows, heads * pad]
  const float* powers;      // [heads][kLightningChunk + 1]: decay^n
  float* state;             // [heads][vdim_pad / 16][dim_pad][16]: as of Control::state_base
  float* chunk_states;      // prompt form: [chunks] of the same
  const Control* control;
  int capacity;
  float* out;               // [rows, heads * vdim_pad]
  TokenDecay token;
};
// At most 16 rows: folds the pending rows into the state, reads it for the step's rows, leaves those pending.
template <typename T>
void launch_lightning_step(const LightningParams& p, cudaStream_t stream, bool pdl);
// A prompt segment in chunks: pending rows and all rows of the segment end up in the state. BF16.
bool lightning_prompt_ok(int dim_pad, int vdim_pad);
void launch_lightning_prompt(const LightningParams& p, cudaStream_t stream, bool pdl, int* launches);

// The mixer's activation row: merged attention splits in front, the normed and gated linear attention behind.
struct MixerFinishParams {
  SizedAttentionParams attention;  // merged if `merge`
  int merge;
  int rows, lin_heads, lin_vdim, lin_vdim_pad;
  const float* lin_out;     // [rows, lin_heads * lin_vdim_pad]
  const void* gate;         // row r at + r * gate_stride: pre-activation of the output gate
  int gate_stride;
  const bf16* norm;         // [lin_heads * lin_vdim_pad]
  float eps, lin_scale;
  void* out;                // the same rows as attention.out
  int out_stride, lin_offset;
};
template <typename T>
void launch_mixer_finish(const MixerFinishParams& p, cudaStream_t stream, bool pdl);

// ---- latent attention (latent_attention.cu) ----
// The cache holds one row per token: the RMS-normed latent [rank_pad] and the rotated key part [rot_pad] shared by all
// heads, zero up to row_pad. A step scores against the latent itself: its queries are taken through the key expansion
// first, and the softmax-weighted latent through the value expansion last.
struct LatentParams {
  void* fused;              // [rows, stride]: q heads of dim_pad + rot_pad | latent [rank_pad] | rotated key | gate
  int rows, stride, latent_at, gate_at;
  int heads, dim_pad, vdim_pad, rank, rank_pad, rot_pad, rot_dims, row_pad;
  float eps;
  const bf16* norm;         // [rank_pad]
  const float2* rotation;   // [capacity][rot_dims / 2] (cos, sin), both times the length factor
  const bf16* expand;       // [heads * dim_pad key rows | heads * vdim_pad value rows][rank_pad]
  void* cache;              // [capacity, row_pad]
  const Control* control;
  int capacity;
  void* query;              // step form: [rows * heads, row_pad], the queries in the space of the cache rows
  void* out;                // [rows, out_stride]: the gated heads; columns beyond them are cleared
  int out_stride;
};
// Latent and rotated key of every row into the cache; with `step` the queries into p.query, otherwise the rotated part
// of the queries in place.
template <typename T>
void launch_latent_prepare(const LatentParams& p, bool step, cudaStream_t stream, bool pdl);
// Split attention of at most 16 rows over the cache: leaves partials in a.scratch (rank_pad values each).
bool latent_attention_ok(int rank_pad, int row_pad, size_t smem_limit);
void launch_latent_attention(const SizedAttentionParams& a, int row_pad, size_t smem_limit, cudaStream_t stream, bool pdl);
// Value expansion and output gate of at most 16 rows. `merge`: from the split attention's partials in a.scratch;
// otherwise from finished latents in a.out [rows, heads * rank_pad].
template <typename T>
void launch_latent_expand(const LatentParams& p, const SizedAttentionParams& a, bool merge, cudaStream_t stream, bool pdl);

// ---- recurrences over one matrix per head (outer_state.cu) ----
// S (key size x value size, FP32): S <- g S, S <- S + k u^T, out = S^T q (+ skip v), after a causal convolution and SiLU
// of q, k and v.
// delta: u = beta (v - S^T k) after the decay, g per key channel, q and k of unit length, beta = sigmoid(step);
// otherwise u = t v with t = softplus(step + bias), g = exp(-rate t) per head.
// State layout as in lightning.cu: [head][slice of 16 values][key dimension][16].
struct OuterStateParams {
  bool delta;
  const void* fused;        // [rows, stride]: q [key_heads * dim_pad] | k | v [heads * vdim_pad] | ...
  int rows, stride, step_at;               // step_at: column of the step pre-activations [heads]
  int heads, key_heads, dim, dim_pad, vdim, vdim_pad, taps;
  const float *conv, *conv_bias;           // [taps][channels], [channels] or null
  void* raw;                               // [raw_rows][channels]: the convolution's inputs by position
  int raw_rows;                            // a power of two
  const void* decay;                       // delta: [rows, decay_stride] pre-activations [heads * dim_pad]
  int decay_stride;
  const float *rate, *bias;                // [heads]; [heads * dim_pad] for delta, else [heads]
  const float* skip;                       // [heads] or null
  float *ring_k, *ring_g, *ring_u;         // [kRingRows][key_heads * dim_pad], [..][heads * dim_pad or heads],
                                           // [..][heads * vdim_pad]
  float *q, *v, *beta;                     // of the step: [rows][key_heads * dim_pad], [rows][heads * vdim_pad], [rows][heads]
  float* state;
  const Control* control;
  int capacity;
  float* out;                              // [rows, heads * vdim_pad]
};
// At most 16 rows, two launches: convolution, decays and rates; the recurrence. Rows stay pending as in lightning.cu:
// the ring keeps their k, g and u, the next step folds those that were kept.
template <typename T>
void launch_outer_prepare(const OuterStateParams& p, cudaStream_t stream, bool pdl);
void launch_outer_step(const OuterStateParams& p, cudaStream_t stream, bool pdl);
// A prompt segment's convolution and SiLU, BF16: out [rows, channels] and, for the delta rule, one over the length of
// every q and k head, inverse [rows, 2 key_heads].
void launch_outer_conv(const OuterStateParams& p, bf16* out, float* inverse, cudaStream_t stream, bool pdl);
// A prompt segment of the delta rule in chunks of 64 tokens (delta_prompt.cu), two launches: pending rows and all rows
// end up in the state.
struct DeltaPromptParams {
  OuterStateParams outer;   // fused (step pre-activations), decay, state, rings, out
  const bf16* conv;         // [rows, channels]
  const float* inverse;     // [rows, 2 key_heads]
  int channels;
  unsigned char* chunks;    // delta_prompt_bytes(rows, heads, dim_pad, vdim_pad)
};
constexpr int kDeltaChunk = 64;
bool delta_prompt_ok(int dim_pad, int vdim_pad);
size_t delta_prompt_bytes(size_t rows, size_t heads, size_t dim_pad, size_t vdim_pad);
void launch_delta_prompt(const DeltaPromptParams& p, cudaStream_t stream, bool pdl);
// RMS norm in `groups` equal parts of the heads' values side by side, weight, and the gate: SiLU ahead of the norm
// (gate_first) or sigmoid behind it.
struct StateFinishParams {
  const float* in;          // [rows, heads * vdim_pad]
  int rows, heads, vdim, vdim_pad, groups;
  const void* gate;         // row r at + r * gate_stride, [heads * vdim_pad]
  int gate_stride;
  bool gate_first;
  const bf16* norm;         // [heads * vdim_pad]
  float eps;
  void* out;
  int out_stride;           // columns beyond the heads' values are cleared
  // after a prompt segment: the convolution inputs of its last tail_rows rows go to the ring
  int tail_rows, tail_stride, channels, raw_rows;
  const void* tail;         // row r at tail + r * tail_stride
  void* raw;
  const Control* control;
  int capacity;
};
template <typename T>
void launch_state_finish(const StateFinishParams& p, cudaStream_t stream, bool pdl);

// ---- gated recurrence (minGRU) ----
struct MinGruParams {
  const void* fused;        // [rows, stride]: gate | candidate | output gate pre-activations, width_pad each
  int rows, stride, width_pad;
  float *ring_gate, *ring_candidate;  // [kRingRows, width_pad]
  float* state;             // [width_pad]: as of Control::state_base
  const Control* control;
  int capacity;
  float* stretches;         // prompt form: [stretches + 1][2 * width_pad]
  void* out;                // [rows, out_stride]; columns beyond width_pad are cleared
  int out_stride;
};
template <typename T>
void launch_min_gru_step(const MinGruParams& p, cudaStream_t stream, bool pdl);
void launch_min_gru_prompt(const MinGruParams& p, cudaStream_t stream, bool pdl);  // two launches

// out[rows, ff] = gated unit of the pair [rows, 2 ff] (clamped).
template <typename T>
void launch_clamped_glu(const T* gate_up, int rows, int ff, float limit, T* out, int multiprocessors,
                        cudaStream_t stream, bool pdl);
// Rows `index[i]` of `source` (row stride in elements) to consecutive rows of `out`.
template <typename T>
void launch_gather_rows(const T* source, const int32_t* index, int count, int stride, T* out, cudaStream_t stream);
// FP32 partial sums -> FP32 sums; cap > 0: cap * tanh(sum / cap). `out` may be `partial`.
void launch_sum_partials(const float* partial, int ksplit, size_t count, float cap, float* out, int multiprocessors,
                         cudaStream_t stream, bool pdl);
// out[rows, out] (FP32) = activation(x (FP32) * W^T (BF16) + bias) with FP32 arithmetic, at most 16 rows of x_stride.
void launch_true32_linear(const float* x, int x_stride, int rows, const PreparedLinear& w, float* out, cudaStream_t stream,
                          bool pdl);
// (cos, sin) of position * frequencies[i], times `length`, computed in double and rounded once.
void launch_rotation_table(float2* table, size_t positions, const double* frequencies, int half, double length,
                           cudaStream_t stream);

// ---- model and session ----
struct LayeredModel {
  struct Layer {
    ei_layer_spec spec{};
    DynamicTanh norm1, norm1b, norm2, norm2b;
    PreparedLinear in, out, gate_up, down;  // fused mixer input, mixer output, feed-forward
    // parallel mixer
    int dim_pad = 0, vdim_pad = 0, lin_dim_pad = 0, lin_vdim_pad = 0, rotation = 0;
    int attention_width = 0, linear_width = 0;  // columns of the mixer's activation row
    const float* sink = nullptr;
    const float* powers = nullptr;
    const bf16* lin_norm = nullptr;
    // gated recurrence
    int width_pad = 0;
    int ff_pad = 0;
    // parallel block: norm weights and the vectors that scale the two results
    const bf16 *norm1_weight = nullptr, *norm2_weight = nullptr, *scale1 = nullptr, *scale2 = nullptr;
    PreparedLinear up;
    // latent attention
    PreparedLinear expand;  // key rows of all heads, then value rows
    int rank_pad = 0, rot_pad = 0, row_pad = 0, latent_at = 0, gate_at = 0;
    const bf16* latent_norm = nullptr;
    // matrix recurrences
    PreparedLinear second;  // second factors of the decay's and the gate's projection, side by side
    int key_heads = 0, channels = 0, raw_rows = 0, step_at = 0, first_at = 0;
    const float *conv = nullptr, *conv_bias = nullptr, *rate = nullptr, *bias = nullptr, *skip = nullptr;
    const bf16* state_norm = nullptr;
    bool outer() const { return spec.mixer == EI_MIXER_STATE_SPACE || spec.mixer == EI_MIXER_CHANNEL_DELTA; }
    bool delta() const { return spec.mixer == EI_MIXER_CHANNEL_DELTA; }
  };
  struct Run {              // one pass through one layer: its own caches and state
    int layer = 0;
    int pass = -1;          // >= 0: the loop pass that starts here
  };
  struct Rotation {
    int dims = 0;
    double base = 0.0, factor = 0.0, original = 0.0, fast = 0.0, slow = 0.0;  // factor 0: no YaRN scaling
    const double* frequencies = nullptr;  // [dims / 2] on the device
    double length = 1.0;
  };
  bool true32 = false, parallel = false;  // parallel: EI_BLOCK_PARALLEL
  int width = 0, residual_stride = 0, normed_stride = 0, vocab_stride = 0, embedding_stride = 0;
  float eps = 0.0f, softcap = 0.0f;
  PairTable pairs;
  const bf16* final_weight = nullptr;
  std::vector<Layer> layers;
  std::vector<Run> runs;
  std::vector<Rotation> rotations;
  const bf16* embedding = nullptr;   // [vocab, embedding_stride]
  const bf16* loop_step = nullptr;   // [times, residual_stride]
  DynamicTanh final_norm;
  PreparedLinear head;
  int max_fused = 0, max_mixed = 0, max_gate_up = 0, max_ff = 0, max_linear = 0, max_rnn = 0;  // widest rows
  int max_second = 0, max_state_keys = 0, max_state_heads = 0;
  size_t max_chunk_state = 0;        // floats of one chunk's state
  // prompt workspace (in ei_model::prompt's arena)
  float *residual = nullptr, *linear_out = nullptr, *chunk_states = nullptr, *stretches = nullptr;
  float *mixed_partial = nullptr, *inverse = nullptr, *decay_totals = nullptr;
  bf16 *second_normed = nullptr, *second = nullptr, *conv_out = nullptr;
  unsigned char* delta_chunks = nullptr;
  int max_channels = 0;
  size_t max_delta_chunks = 0;       // bytes for a whole segment
  // Latent attention over a prompt: keys and values of every cached token of one layer, grown when a longer history
  // comes by.
  bf16* expanded = nullptr;
  size_t expanded_bytes = 0, max_expand = 0;  // max_expand: widest row
  LayeredModel() = default;
  LayeredModel(const LayeredModel&) = delete;
  ~LayeredModel() {
    if (expanded) cudaFree(expanded);
  }
};

struct LayeredSession {
  struct Run {
    void *k_cache = nullptr, *v_cache = nullptr;
    void *ring_k = nullptr, *ring_v = nullptr;          // activation type
    float *ring_gate = nullptr, *ring_candidate = nullptr;
    void *latent = nullptr, *raw = nullptr;             // activation type
    float *ring_key = nullptr, *ring_decay = nullptr, *ring_write = nullptr;
    float* state = nullptr;
  };
  std::vector<Run> runs;
  std::vector<float2*> rotations;
  size_t token_rows = 0;             // cache rows allocated (the capacity, whole tiles)
  float *residual = nullptr, *linear_out = nullptr, *logits = nullptr, *head_partial = nullptr;
  void *normed = nullptr, *fused = nullptr, *mixed = nullptr, *gate_up = nullptr, *act = nullptr, *head_rows = nullptr;
  float* mixed_partial = nullptr;    // a parallel block's mixer sums, until its feed-forward's are there
  void *second_normed = nullptr, *second = nullptr, *latent_query = nullptr, *latent_out = nullptr;
  float *state_q = nullptr, *state_v = nullptr, *state_beta = nullptr;
  uint32_t* history = nullptr;       // [capacity]: the token of every position
  float* tap = nullptr;              // caller's device buffer [runs][tap_rows][width], or null
  size_t tap_rows = 0;
};

// Builds `model` (device and limits already set) from the description and the checkpoint's tensors.
void create_layered_model(ei_model& model, const ei_layered_config& config, const ei_layer_spec* layers,
                          const ei_named_tensor* tensors, size_t count);
void create_layered_session(ei_session& s);
void ensure_layered_workspace(ei_model& model);
// Room for the expanded keys and values of `tokens` tokens; the caller holds the prompt workspace and its stream is idle.
void ensure_expanded(ei_model& model, size_t tokens);
// One forward of at most 16 rows at the device-side context length / of a prompt segment. The segment leaves the
// normed rows in the prompt workspace; the vocabulary head runs in enqueue_layered_head over gathered rows.
void enqueue_layered_step(ei_session& s, int rows, StepKind kind);
// `context`: the context length the segment starts at, as the device will find it.
void enqueue_layered_segment(ei_session& s, int rows, size_t context);
// FP32 logits of `count` <= 16 rows of the segment (indices on the device) into the session's logits; with `greedy`
// the greedy token of row 0 goes to s.targets[0].
void enqueue_layered_head(ei_session& s, const int32_t* device_rows, int count, bool greedy);

}  // namespace ei
