// Decoders described layer by layer: weights, caches and state, and the two forms of a forward.
//
// A step (at most 16 rows: decode, verify, a short portion) runs per layer, with programmatic dependent launch:
//   parallel mixer   fused projection -> heads prepared, K / V appended -> split attention -> linear attention step ->
//                    merge + gate -> output projection (FP32 sums) -> join
//   gated recurrence fused projection -> recurrence step -> output projection (FP32 sums) -> join
//   feed-forward     gate|up with the gated unit in the epilogue -> down (FP32 sums) -> join
// where a join finishes one sublayer (norm after, residual add, what a loop pass adds) and starts the next (norm
// before). A prompt segment runs the same sequence over all its rows on the prompt GEMM, whole-history attention and
// the chunked forms of the recurrences. A model in true 32-bit runs every token through the step form.
#include "layered.cuh"

#include <cmath>
#include <cstring>
#include <limits>
#include <set>

namespace ei {
namespace {

int round_up(size_t value, int step) {
  const size_t rounded = (value + step - 1) / step * step;
  if (rounded > size_t(std::numeric_limits<int>::max() / 4)) throw std::invalid_argument("Layered decoder: a size is out of range");
  return int(rounded);
}

// Places the tensors in one arena. `base` null: only the sizes are added up and the shapes checked.
struct Placement {
  std::map<std::string, const ei_named_tensor*> tensors;
  std::set<std::string> used;
  unsigned char* base = nullptr;
  size_t offset = 0;

  const ei_named_tensor& find(const std::string& name, size_t rows, size_t columns) {
    auto it = tensors.find(name);
    if (it == tensors.end()) throw std::invalid_argument("Layered decoder weight not found: " + name);
    const ei_named_tensor& t = *it->second;
    const bool fits = columns ? t.rank == 2 && t.shape[0] == rows && t.shape[1] == columns : t.rank == 1 && t.shape[0] == rows;
    if (!fits || t.kind != 0) throw std::invalid_argument("Layered decoder weight shape mismatch: " + name);
    used.insert(name);
    return t;
  }
  template <typename T>
  T* reserve(size_t count) {
    T* at = base ? reinterpret_cast<T*>(base + offset) : nullptr;
    offset += aligned(count * sizeof(T));
    return at;
  }
  // `rows` x `columns` of a BF16 source with row pitch source_pitch into a destination with pitch pitch.
  void copy(bf16* to, size_t pitch, const void* from, size_t source_pitch, size_t rows, size_t columns) {
    if (base) EI_CUDA(cudaMemcpy2D(to, pitch * 2, from, source_pitch * 2, columns * 2, rows, cudaMemcpyDefault));
  }
  template <typename T>
  const T* host_values(const std::vector<T>& values) {
    T* at = reserve<T>(values.size());
    if (base) EI_CUDA(cudaMemcpy(at, values.data(), values.size() * sizeof(T), cudaMemcpyHostToDevice));
    return at;
  }
  std::vector<float> read(const ei_named_tensor& t) {
    std::vector<uint16_t> bits(t.shape[0]);
    std::vector<float> values(t.shape[0]);
    EI_CUDA(cudaMemcpy(bits.data(), t.data, bits.size() * 2, cudaMemcpyDefault));
    for (size_t i = 0; i < bits.size(); ++i) {
      const uint32_t wide = uint32_t(bits[i]) << 16;
      std::memcpy(&values[i], &wide, 4);
    }
    return values;
  }
  const bf16* vector(const std::string& name, size_t width, size_t pad) {
    const ei_named_tensor& t = find(name, width, 0);
    bf16* at = reserve<bf16>(pad);
    copy(at, width, t.data, width, 1, width);
    return at;
  }
  const bf16* matrix(const std::string& name, size_t rows, size_t columns, size_t row_pad, size_t pitch) {
    const ei_named_tensor& t = find(name, rows, columns);
    bf16* at = reserve<bf16>(row_pad * pitch);
    copy(at, pitch, t.data, columns, rows, columns);
    return at;
  }
  DynamicTanh norm(const std::string& name, size_t width, size_t pad) {
    DynamicTanh n;
    n.weight = vector(name, width, pad);
    n.bias = vector(name + ".b", width, pad);
    const ei_named_tensor& alpha = find(name + ".alpha", 1, 0);
    if (base) n.alpha = read(alpha)[0];
    return n;
  }
  // A zeroed linear [out, in] to be filled section by section.
  PreparedLinear linear(int in, int out, bf16** weights) {
    PreparedLinear l;
    l.in = in;
    l.out = out;
    *weights = reserve<bf16>(size_t(out) * in);
    l.dense = *weights;
    l.bytes = size_t(out) * in * 2;
    return l;
  }
  // Output rows of `heads` heads of `size` features, `pad` rows apart; returns the row behind them.
  int rows_of(bf16* weights, int pitch, int row, const std::string& name, int heads, int size, int pad, size_t inputs) {
    const ei_named_tensor& t = find(name, size_t(heads) * size, inputs);
    if (base)
      for (int h = 0; h < heads; ++h)
        copy(weights + (size_t(row) + size_t(h) * pad) * pitch, pitch,
             static_cast<const bf16*>(t.data) + size_t(h) * size * inputs, inputs, size, inputs);
    return row + heads * pad;
  }
  // Input columns of `heads` heads of `size` values, `pad` columns apart.
  void columns_of(bf16* weights, int pitch, int column, const std::string& name, int heads, int size, int pad, size_t outputs) {
    const ei_named_tensor& t = find(name, outputs, size_t(heads) * size);
    if (base)
      for (int h = 0; h < heads; ++h)
        copy(weights + column + size_t(h) * pad, pitch, static_cast<const bf16*>(t.data) + size_t(h) * size,
             size_t(heads) * size, outputs, size);
  }
};

void validate_layer(const ei_layer_spec& l) {
  auto in_range = [](uint32_t v, uint32_t most) { return v >= 1 && v <= most; };
  constexpr uint32_t kMany = 1u << 20;
  if (l.mixer == EI_MIXER_MIN_GRU) {
    if (!in_range(l.rnn_width, kMany)) throw std::invalid_argument("Layered decoder: invalid recurrence width");
  } else if (l.mixer == EI_MIXER_PARALLEL) {
    if (!in_range(l.heads, 4096) || !in_range(l.kv_heads, 4096) || l.heads % l.kv_heads || !in_range(l.dim, kMaxHeadDim) ||
        !in_range(l.vdim, kMaxHeadDim) || l.rot_dims > l.dim || l.rot_dims % 2 || !(l.rot_base > 0.0) || !std::isfinite(l.scale))
      throw std::invalid_argument("Layered decoder: invalid attention sizes (head sizes are limited to 512)");
    if (!in_range(l.lin_heads, 4096) || !in_range(l.lin_dim, kMaxHeadDim) || !in_range(l.lin_vdim, kMaxHeadDim) || !l.decay)
      throw std::invalid_argument("Layered decoder: invalid linear attention sizes (head sizes are limited to 512)");
    if (!std::isfinite(l.left_scale) || !std::isfinite(l.right_scale))
      throw std::invalid_argument("Layered decoder: invalid mixer scale");
  } else {
    throw std::invalid_argument("Layered decoder: unknown mixer");
  }
  if (l.mlp != EI_MLP_NONE && (l.mlp != EI_MLP_CLAMPED_GLU || !in_range(l.ff, kMany) || std::isnan(l.limit)))
    throw std::invalid_argument("Layered decoder: invalid feed-forward");
}

void place(ei_model& model, const ei_layered_config& c, const ei_layer_spec* specs, Placement& at) {
  LayeredModel& m = *model.layered;
  const size_t W = c.width, V = c.vocab_size;
  const int R = m.residual_stride, K = m.normed_stride;
  at.offset = 0;
  m.layers.assign(c.n_layers, {});
  m.rotations.clear();
  m.embedding = at.matrix("embed", V, W, V, R);
  if (c.loop_times) m.loop_step = at.matrix("loop.step", c.loop_times, W, c.loop_times, R);
  m.final_norm = at.norm("final.norm", W, R);
  bf16* weights = nullptr;
  m.head = at.linear(K, m.vocab_stride, &weights);
  at.rows_of(weights, K, 0, "head", 1, int(V), int(V), W);
  for (size_t i = 0; i < c.n_layers; ++i) {
    const std::string p = "l" + std::to_string(i) + ".", mix = p + "mix.";
    LayeredModel::Layer& L = m.layers[i];
    const ei_layer_spec& s = L.spec = specs[i];
    L.spec.decay = nullptr;
    L.norm1 = at.norm(p + "norm1", W, R);
    L.norm1b = at.norm(p + "norm1b", W, R);
    if (s.mixer == EI_MIXER_MIN_GRU) {
      const int width = int(s.rnn_width);
      L.width_pad = round_up(width, 16);
      L.in = at.linear(K, 3 * L.width_pad, &weights);
      int row = at.rows_of(weights, K, 0, mix + "z", 1, width, L.width_pad, W);
      row = at.rows_of(weights, K, row, mix + "x", 1, width, L.width_pad, W);
      at.rows_of(weights, K, row, mix + "g", 1, width, L.width_pad, W);
      bf16* bias = at.reserve<bf16>(L.in.out);
      at.copy(bias, width, at.find(mix + "z.b", width, 0).data, width, 1, width);
      at.copy(bias + L.width_pad, width, at.find(mix + "x.b", width, 0).data, width, 1, width);
      L.in.bias = bias;
      L.out = at.linear(round_up(width, 64), R, &weights);
      at.columns_of(weights, L.out.in, 0, mix + "o", 1, width, L.width_pad, W);
    } else {
      const std::string left = mix + "left.", right = mix + "right.";
      L.dim_pad = round_up(s.dim, 16);
      L.vdim_pad = round_up(s.vdim, 16);
      L.lin_dim_pad = round_up(s.lin_dim, 16);
      L.lin_vdim_pad = round_up(s.lin_vdim, 16);
      L.attention_width = int(s.heads) * L.vdim_pad;
      L.linear_width = int(s.lin_heads) * L.lin_vdim_pad;
      const int H = int(s.heads), G = int(s.kv_heads), N = int(s.lin_heads);
      L.in = at.linear(K, (H + G) * L.dim_pad + G * L.vdim_pad + 2 * N * (L.lin_dim_pad + L.lin_vdim_pad), &weights);
      int row = at.rows_of(weights, K, 0, left + "q", H, int(s.dim), L.dim_pad, W);
      row = at.rows_of(weights, K, row, left + "k", G, int(s.dim), L.dim_pad, W);
      row = at.rows_of(weights, K, row, left + "v", G, int(s.vdim), L.vdim_pad, W);
      row = at.rows_of(weights, K, row, right + "q", N, int(s.lin_dim), L.lin_dim_pad, W);
      row = at.rows_of(weights, K, row, right + "k", N, int(s.lin_dim), L.lin_dim_pad, W);
      row = at.rows_of(weights, K, row, right + "v", N, int(s.lin_vdim), L.lin_vdim_pad, W);
      at.rows_of(weights, K, row, right + "g", N, int(s.lin_vdim), L.lin_vdim_pad, W);
      L.out = at.linear(round_up(L.attention_width + L.linear_width, 64), R, &weights);
      at.columns_of(weights, L.out.in, 0, left + "o", H, int(s.vdim), L.vdim_pad, W);
      at.columns_of(weights, L.out.in, L.attention_width, right + "o", N, int(s.lin_vdim), L.lin_vdim_pad, W);
      L.sink = at.host_values(at.base ? at.read(at.find(left + "sink", H, 0))
                                      : (at.find(left + "sink", H, 0), std::vector<float>(H)));
      bf16* norm = at.reserve<bf16>(L.linear_width);
      at.copy(norm, L.lin_vdim_pad, at.find(right + "norm", size_t(N) * s.lin_vdim, 0).data, s.lin_vdim, N, s.lin_vdim);
      L.lin_norm = norm;
      std::vector<float> powers;
      for (int h = 0; h < N; ++h)
        for (int n = 0; n <= kLightningChunk; ++n) powers.push_back(float(std::pow(specs[i].decay[h], n)));
      L.powers = at.host_values(powers);
      for (L.rotation = 0; L.rotation < int(m.rotations.size()); ++L.rotation)
        if (m.rotations[L.rotation].dims == int(s.rot_dims) && m.rotations[L.rotation].base == s.rot_base) break;
      if (L.rotation == int(m.rotations.size())) m.rotations.push_back({int(s.rot_dims), s.rot_base});
    }
    if (s.mlp != EI_MLP_NONE) {
      L.norm2 = at.norm(p + "norm2", W, R);
      L.norm2b = at.norm(p + "norm2b", W, R);
      L.ff_pad = round_up(s.ff, 64);
      L.gate_up = at.linear(K, 2 * L.ff_pad, &weights);
      L.gate_up.glu = kGluClamped;
      L.gate_up.glu_limit = float(s.limit);
      at.rows_of(weights, K, 0, p + "mlp.gate", 1, int(s.ff), L.ff_pad, W);
      at.rows_of(weights, K, L.ff_pad, p + "mlp.up", 1, int(s.ff), L.ff_pad, W);
      L.down = at.linear(L.ff_pad, R, &weights);
      at.columns_of(weights, L.ff_pad, 0, p + "mlp.down", 1, int(s.ff), L.ff_pad, W);
    }
  }
}

size_t partial_floats(const PreparedLinear& w) {
  const int units = w.in / 64;
  const int slices = std::max(1, (units + kGemmWarps * 4 - 1) / (kGemmWarps * 4));
  return size_t(slices) * kMaxRows * w.out;
}


// Step-form projections. The result of `store` is in the activation type, with bias; `sums` leaves FP32 sums in
// s.partial and returns the number of K slices.
template <typename T>
struct StepLinear;
template <>
struct StepLinear<bf16> {
  static int sums(ei_session& s, const PreparedLinear& w, const bf16* x, int rows) {
    int ksplit = 1;
    run_linear(s, w, x, rows, kEpiPartial, nullptr, 0, true, &ksplit);
    return ksplit;
  }
  static void store(ei_session& s, const PreparedLinear& w, const bf16* x, int rows, bf16* out) {
    if (has_plan(s, w, rows, kEpiStore)) {
      run_linear(s, w, x, rows, kEpiStore, out, w.out, true);
      return;
    }
    const int ksplit = sums(s, w, x, rows);
    tick(s);
    launch(splitk_store_kernel, dim3(std::min(s.model->multiprocessors * 8, (rows * w.out + 255) / 256)), dim3(256), 0,
           s.stream, true, (const float*)s.partial, ksplit, rows, w.out, w.bias, out, w.out);
  }
  static void gated(ei_session& s, const PreparedLinear& w, const bf16* x, int rows, bf16* pair, bf16* out) {
    if (has_plan(s, w, rows, kEpiSiluPair)) {
      run_linear(s, w, x, rows, kEpiSiluPair, out, w.out / 2, true);
      return;
    }
    store(s, w, x, rows, pair);
    tick(s);
    launch_clamped_glu<bf16>(pair, rows, w.out / 2, w.glu_limit, out, s.model->multiprocessors, s.stream, true);
  }
};
template <>
struct StepLinear<float> {
  static int sums(ei_session& s, const PreparedLinear& w, const float* x, int rows) {
    tick(s);
    launch_true32_linear(x, rows, w, s.partial, s.stream, true);
    return 1;
  }
  static void store(ei_session& s, const PreparedLinear& w, const float* x, int rows, float* out) {
    tick(s);
    launch_true32_linear(x, rows, w, out, s.stream, true);
  }
  static void gated(ei_session& s, const PreparedLinear& w, const float* x, int rows, float* pair, float* out) {
    store(s, w, x, rows, pair);
    tick(s);
    launch_clamped_glu<float>(pair, rows, w.out / 2, w.glu_limit, out, s.model->multiprocessors, s.stream, true);
  }
};

// The vocabulary head over at most 16 rows: FP32 logits in the session; with `parts` the argmax partials too.
template <typename T>
void run_head(ei_session& s, const T* rows_in, int rows, int* parts) {
  const LayeredModel& m = *s.model->layered;
  LayeredSession& L = *s.layered;
  float* keep = s.partial;
  s.partial = L.head_partial ? L.head_partial : L.logits;
  int ksplit = 1;
  try {
    ksplit = StepLinear<T>::sums(s, m.head, rows_in, rows);
  } catch (...) {
    s.partial = keep;
    throw;
  }
  s.partial = keep;
  if (L.head_partial) {
    tick(s);
    launch_sum_partials(L.head_partial, ksplit, size_t(rows) * m.vocab_stride, L.logits, s.model->multiprocessors, s.stream, true);
  }
  if (!parts) return;
  const size_t vocab = s.model->config.vocab_size;
  *parts = std::min(kSampleMaxParts, sample_partial_blocks(vocab, s.model->multiprocessors));
  tick(s);
  launch_argmax_partials_f32(L.logits, rows, vocab, m.vocab_stride, s.best_value, s.best_index, *parts, s.stream, true);
}

// What a step and a prompt segment have in common: the fused sequence over buffers of one activation type.
struct Buffers {
  int rows;
  const uint32_t* tokens;  // of the rows, for the loop's embedding injection
  float *residual, *linear_out;
  void *normed, *fused, *mixed, *gate_up, *act;
};

DynamicTanh norm_ahead(const LayeredModel& m, size_t run) {
  return run < m.runs.size() ? m.layers[m.runs[run].layer].norm1 : m.final_norm;
}

SublayerJoinParams join_params(const ei_session& s, const Buffers& b, const float* partial, int ksplit) {
  const LayeredModel& m = *s.model->layered;
  SublayerJoinParams j{};
  j.partial = partial;
  j.ksplit = ksplit;
  j.rows = b.rows;
  j.residual = b.residual;
  j.residual_stride = m.residual_stride;
  j.normed = b.normed;
  j.normed_stride = m.normed_stride;
  return j;
}

// The join that ends layer run `run`: inspection copy, what the next pass of the loop adds, the next norm.
void end_of_run(const ei_session& s, const Buffers& b, size_t run, SublayerJoinParams& j) {
  const LayeredModel& m = *s.model->layered;
  const LayeredSession& L = *s.layered;
  if (L.tap) {
    j.tap = L.tap + run * L.tap_rows * m.width;
    j.tap_width = m.width;
  }
  if (run + 1 < m.runs.size() && m.runs[run + 1].pass >= 0) {
    if (m.runs[run + 1].pass > 0) {
      j.inject.tokens = b.tokens;
      j.inject.table = m.embedding;
      j.inject.vocab = int(s.model->config.vocab_size);
    }
    j.inject.vector = m.loop_step + size_t(m.runs[run + 1].pass) * m.residual_stride;
  }
  j.before = norm_ahead(m, run + 1);
}

template <typename T>
void enqueue_embed(ei_session& s, const Buffers& b, const EmbedParams& token) {
  const LayeredModel& m = *s.model->layered;
  LayeredEmbedParams e{};
  e.token = token;
  e.table = m.embedding;
  if (m.runs[0].pass >= 0) e.vector = m.loop_step + size_t(m.runs[0].pass) * m.residual_stride;
  e.norm = norm_ahead(m, 0);
  e.residual = b.residual;
  e.residual_stride = m.residual_stride;
  e.normed = b.normed;
  e.normed_stride = m.normed_stride;
  tick(s);
  launch_layered_embed<T>(e, s.stream, false);
}

MixerPrepareParams prepare_params(const ei_session& s, const LayeredModel::Layer& l, const LayeredSession::Run& r,
                                  const Buffers& b, bool pending) {
  MixerPrepareParams p{};
  p.fused = b.fused;
  p.rows = b.rows;
  p.stride = l.in.out;
  p.heads = int(l.spec.heads);
  p.kv_heads = int(l.spec.kv_heads);
  p.dim = int(l.spec.dim);
  p.vdim = int(l.spec.vdim);
  p.dim_pad = l.dim_pad;
  p.vdim_pad = l.vdim_pad;
  p.rot_dims = int(l.spec.rot_dims);
  p.eps = s.model->layered->eps;
  p.rotation = s.layered->rotations[l.rotation];
  p.control = s.control;
  p.capacity = int(s.capacity);
  p.k_cache = r.k_cache;
  p.v_cache = r.v_cache;
  p.lin_heads = int(l.spec.lin_heads);
  p.lin_dim_pad = l.lin_dim_pad;
  p.lin_vdim_pad = l.lin_vdim_pad;
  if (pending) {
    p.ring_k = r.ring_k;
    p.ring_v = r.ring_v;
  }
  return p;
}

SizedAttentionParams attention_params(ei_session& s, const LayeredModel::Layer& l, const LayeredSession::Run& r,
                                      const Buffers& b) {
  SizedAttentionParams a{};
  a.q = b.fused;
  a.q_stride = l.in.out;
  a.k = r.k_cache;
  a.v = r.v_cache;
  a.rows = b.rows;
  a.heads = int(l.spec.heads);
  a.kv_heads = int(l.spec.kv_heads);
  a.dim_pad = l.dim_pad;
  a.vdim_pad = l.vdim_pad;
  a.scale = float(l.spec.scale);
  a.out_scale = float(l.spec.left_scale);
  a.sink = l.sink;
  a.device_offset = &s.control->context;
  a.capacity = int(s.capacity);
  a.chunk = s.attention_chunk;
  a.max_splits = s.attention_splits;
  a.scratch = s.attention_scratch;
  a.out = b.mixed;
  a.out_stride = l.out.in;
  a.status = &s.control->status;
  if (s.inject_attention_polls) {
    a.wait_limit = s.inject_attention_polls;
    a.fault_tx = 16;
    s.inject_attention_polls = 0;  // one launch only
  }
  return a;
}

template <typename T>
LightningParams lightning_params(const ei_session& s, const LayeredModel::Layer& l, const LayeredSession::Run& r,
                                 const Buffers& b) {
  LightningParams p{};
  const int H = int(l.spec.heads), G = int(l.spec.kv_heads), N = int(l.spec.lin_heads);
  const T* q = static_cast<const T*>(b.fused) + (H + G) * l.dim_pad + G * l.vdim_pad;
  p.q = q;
  p.k = q + N * l.lin_dim_pad;
  p.v = q + 2 * N * l.lin_dim_pad;
  p.stride = l.in.out;
  p.rows = b.rows;
  p.heads = N;
  p.dim_pad = l.lin_dim_pad;
  p.vdim_pad = l.lin_vdim_pad;
  p.ring_k = r.ring_k;
  p.ring_v = r.ring_v;
  p.powers = l.powers;
  p.state = r.state;
  p.chunk_states = s.model->layered->chunk_states;
  p.control = s.control;
  p.capacity = int(s.capacity);
  p.out = b.linear_out;
  return p;
}

template <typename T>
MixerFinishParams finish_params(const ei_session& s, const LayeredModel::Layer& l, const Buffers& b,
                                const SizedAttentionParams& a, bool merge) {
  MixerFinishParams f{};
  const int H = int(l.spec.heads), G = int(l.spec.kv_heads), N = int(l.spec.lin_heads);
  f.attention = a;
  f.merge = merge;
  f.rows = b.rows;
  f.lin_heads = N;
  f.lin_vdim = int(l.spec.lin_vdim);
  f.lin_vdim_pad = l.lin_vdim_pad;
  f.lin_out = b.linear_out;
  f.gate = static_cast<const T*>(b.fused) + (H + G) * l.dim_pad + G * l.vdim_pad + N * (2 * l.lin_dim_pad + l.lin_vdim_pad);
  f.gate_stride = l.in.out;
  f.norm = l.lin_norm;
  f.eps = s.model->layered->eps;
  f.lin_scale = float(l.spec.right_scale);
  f.out = b.mixed;
  f.out_stride = l.out.in;
  f.lin_offset = l.attention_width;
  return f;
}

template <typename T>
MinGruParams min_gru_params(const ei_session& s, const LayeredModel::Layer& l, const LayeredSession::Run& r,
                            const Buffers& b) {
  MinGruParams g{};
  g.fused = b.fused;
  g.rows = b.rows;
  g.stride = l.in.out;
  g.width_pad = l.width_pad;
  g.ring_gate = r.ring_gate;
  g.ring_candidate = r.ring_candidate;
  g.state = r.state;
  g.stretches = s.model->layered->stretches;
  g.control = s.control;
  g.capacity = int(s.capacity);
  g.out = b.mixed;
  g.out_stride = l.out.in;
  return g;
}

template <typename T>
void enqueue_step_as(ei_session& s, int rows, StepKind kind) {
  const LayeredModel& m = *s.model->layered;
  LayeredSession& L = *s.layered;
  const bool pdl = true;
  const size_t before = s.launches;
  const Buffers b{rows, s.step_tokens, L.residual, L.linear_out, L.normed, L.fused, L.mixed, L.gate_up, L.act};
  EmbedParams token{};
  token.tokens = kind == kVerifyDevice ? nullptr : s.tokens;
  token.source = kind == kVerifyDevice ? s.draft_source : nullptr;
  token.control = s.control;
  token.step_tokens = s.step_tokens;
  token.vocab = int(s.model->config.vocab_size);
  token.rows = rows;
  token.capacity = int(s.capacity);
  enqueue_embed<T>(s, b, token);

  for (size_t run = 0; run < m.runs.size(); ++run) {
    const LayeredModel::Layer& l = m.layers[m.runs[run].layer];
    const LayeredSession::Run& r = L.runs[run];
    StepLinear<T>::store(s, l.in, static_cast<const T*>(b.normed), rows, static_cast<T*>(b.fused));
    if (l.spec.mixer == EI_MIXER_MIN_GRU) {
      tick(s);
      launch_min_gru_step<T>(min_gru_params<T>(s, l, r, b), s.stream, pdl);
    } else {
      tick(s);
      launch_mixer_prepare<T>(prepare_params(s, l, r, b, true), s.stream, pdl);
      const SizedAttentionParams a = attention_params(s, l, r, b);
      const bool tiled = !m.true32 && sized_attention_ok(l.dim_pad, l.vdim_pad);
      tick(s);
      if (tiled)
        launch_sized_attention_step(a, s.stream, pdl);
      else
        launch_plain_attention<T>(a, s.stream, pdl);
      tick(s);
      launch_lightning_step<T>(lightning_params<T>(s, l, r, b), s.stream, pdl);
      tick(s);
      launch_mixer_finish<T>(finish_params<T>(s, l, b, a, tiled), s.stream, pdl);
    }
    int ksplit = StepLinear<T>::sums(s, l.out, static_cast<const T*>(b.mixed), rows);
    SublayerJoinParams j = join_params(s, b, s.partial, ksplit);
    j.after = l.norm1b;
    if (l.spec.mlp == EI_MLP_NONE)
      end_of_run(s, b, run, j);
    else
      j.before = l.norm2;
    tick(s);
    launch_sublayer_join<T>(j, s.stream, pdl);
    if (l.spec.mlp == EI_MLP_NONE) continue;
    StepLinear<T>::gated(s, l.gate_up, static_cast<const T*>(b.normed), rows, static_cast<T*>(b.gate_up), static_cast<T*>(b.act));
    ksplit = StepLinear<T>::sums(s, l.down, static_cast<const T*>(b.act), rows);
    j = join_params(s, b, s.partial, ksplit);
    j.after = l.norm2b;
    end_of_run(s, b, run, j);
    tick(s);
    launch_sublayer_join<T>(j, s.stream, pdl);
  }

  if (kind == kCommitAllNoHead) {
    enqueue_commit(s, rows, false);
  } else {
    int parts = 0;
    run_head<T>(s, static_cast<const T*>(b.normed), rows, &parts);
    tick(s);
    if (kind == kCommitAllWithHead) {
      launch_finalize(s.best_value, s.best_index, parts, rows, s.targets, nullptr, nullptr, nullptr, nullptr, nullptr,
                      s.stream, pdl);
      enqueue_commit(s, rows, false);
    } else {
      launch_finalize(s.best_value, s.best_index, parts, rows, s.targets, s.step_tokens, s.control, nullptr, nullptr,
                      nullptr, s.stream, pdl, s.token_sink);
    }
  }
  s.launches_per_step[rows] = s.launches - before;
}

}  // namespace

void create_layered_model(ei_model& model, const ei_layered_config& c, const ei_layer_spec* specs,
                          const ei_named_tensor* tensors, size_t count) {
  auto positive = [](uint64_t v, uint64_t most) { return v >= 1 && v <= most; };
  constexpr uint64_t kMany = 1u << 24;
  if (!positive(c.vocab_size, kMany) || !positive(c.width, 1u << 18) || !positive(c.n_layers, 1u << 16) ||
      !positive(c.max_position_embeddings, 1u << 30) || !std::isfinite(c.norm_eps) || c.norm_eps < 0.0)
    throw std::invalid_argument("Layered decoder: sizes must be positive and in range");
  if (c.loop_times && (c.loop_times > 65536 || c.loop_start >= c.loop_stop || c.loop_stop > c.n_layers))
    throw std::invalid_argument("Layered decoder: the loop must span existing layers");
  for (size_t i = 0; i < c.n_layers; ++i) validate_layer(specs[i]);

  model.layered = std::make_shared<LayeredModel>();
  LayeredModel& m = *model.layered;
  m.true32 = c.true32 != 0;
  m.width = int(c.width);
  m.residual_stride = round_up(c.width, 16);
  m.normed_stride = round_up(c.width, 64);
  m.vocab_stride = round_up(c.vocab_size, 16);
  m.eps = float(c.norm_eps);
  model.config.vocab_size = c.vocab_size;
  model.config.n_layers = c.n_layers;
  model.config.hidden_size = c.width;
  model.config.max_position_embeddings = c.max_position_embeddings;
  model.config.bos_token_id = c.bos_token_id;
  model.config.eos_token_id = c.eos_token_id;
  model.config.rms_norm_eps = m.eps;

  const auto range = [&](uint64_t from, uint64_t to, int pass) {
    for (uint64_t i = from; i < to; ++i) m.runs.push_back({int(i), pass >= 0 && i == from ? pass : -1});
  };
  if (c.loop_times) {
    range(0, c.loop_start, -1);
    for (uint64_t t = 0; t < c.loop_times; ++t) range(c.loop_start, c.loop_stop, int(t));
    range(c.loop_stop, c.n_layers, -1);
  } else {
    range(0, c.n_layers, -1);
  }

  Placement placement;
  for (size_t i = 0; i < count; ++i) {
    const ei_named_tensor& t = tensors[i];
    if (!t.name || !t.data || t.rank < 1 || t.rank > 2) throw std::invalid_argument("Empty or malformed layered decoder weight");
    if (!placement.tensors.emplace(t.name, &t).second)
      throw std::invalid_argument(std::string("Duplicate layered decoder weight: ") + t.name);
  }
  place(model, c, specs, placement);
  for (const auto& entry : placement.tensors)
    if (!placement.used.count(entry.first))
      throw std::invalid_argument("Unexpected layered decoder weight: " + entry.first);
  model.arena_bytes = placement.offset;
  EI_CUDA(cudaMalloc(reinterpret_cast<void**>(&model.arena), placement.offset));
  try {
    EI_CUDA(cudaMemset(model.arena, 0, placement.offset));
    placement.base = model.arena;
    place(model, c, specs, placement);
    EI_CUDA(cudaDeviceSynchronize());
  } catch (...) {
    cudaFree(model.arena);
    model.arena = nullptr;
    throw;
  }

  model.weight_bytes = m.head.bytes;
  for (const auto& run : m.runs) {
    const auto& l = m.layers[run.layer];
    model.weight_bytes += l.in.bytes + l.out.bytes + l.gate_up.bytes + l.down.bytes;
  }
  model.prompt_ready = !m.true32;
  for (const auto& l : m.layers) {
    m.max_fused = std::max(m.max_fused, l.in.out);
    m.max_mixed = std::max(m.max_mixed, l.out.in);
    m.max_gate_up = std::max(m.max_gate_up, l.gate_up.out);
    m.max_ff = std::max(m.max_ff, l.ff_pad);
    m.max_linear = std::max(m.max_linear, l.linear_width);
    m.max_rnn = std::max(m.max_rnn, l.width_pad);
    if (l.spec.mixer == EI_MIXER_PARALLEL) {
      m.max_chunk_state = std::max(m.max_chunk_state, size_t(l.linear_width) * l.lin_dim_pad);
      model.prompt_ready = model.prompt_ready && sized_attention_ok(l.dim_pad, l.vdim_pad) &&
                           lightning_prompt_ok(l.lin_dim_pad, l.lin_vdim_pad);
    }
    model.prompt_ready = model.prompt_ready && prompt_linear_ok(l.in) && prompt_linear_ok(l.out) &&
                         (l.spec.mlp == EI_MLP_NONE || (prompt_linear_ok(l.gate_up) && prompt_linear_ok(l.down)));
  }
}

void create_layered_session(ei_session& s) {
  const ei_model& model = *s.model;
  const LayeredModel& m = *model.layered;
  s.layered = std::make_shared<LayeredSession>();
  LayeredSession& L = *s.layered;
  const size_t T = m.true32 ? 4 : 2;  // bytes of an activation
  s.attention_chunk = attention_chunk_for(s.capacity);
  s.attention_splits = int((s.capacity + s.attention_chunk - 1) / s.attention_chunk);
  L.token_rows = (s.capacity + 63) / 64 * 64;
  size_t partial = 0, scratch = 0;
  for (const auto& l : m.layers) {
    for (const PreparedLinear* w : {&l.in, &l.out, &l.gate_up, &l.down}) partial = std::max(partial, partial_floats(*w));
    if (l.spec.mixer == EI_MIXER_PARALLEL)
      scratch = std::max(scratch, sized_attention_scratch_bytes(kMaxRows, l.spec.heads, l.vdim_pad, s.capacity));
  }
  const size_t head_partial = partial_floats(m.head) > size_t(kMaxRows) * m.vocab_stride ? partial_floats(m.head) : 0;

  std::vector<std::pair<void**, size_t>> wanted;
  size_t total = 0;
  auto take = [&](auto*& pointer, size_t bytes) {
    wanted.emplace_back(reinterpret_cast<void**>(&pointer), total);
    total += aligned(std::max<size_t>(bytes, 1));
  };
  take(s.partial, partial * sizeof(float));
  take(s.attention_scratch, scratch);
  take(s.best_value, size_t(kSampleMaxParts) * 16 * sizeof(float));
  take(s.best_index, size_t(kSampleMaxParts) * 16 * sizeof(int));
  take(s.tokens, kMaxRows * 4);
  take(s.step_tokens, kMaxRows * 4);
  take(s.targets, kMaxRows * 4);
  take(s.control, sizeof(Control));
  take(s.draft_source, sizeof(DraftSource));
  take(s.token_sink, sizeof(TokenSink));
  take(L.residual, size_t(kMaxRows) * m.residual_stride * sizeof(float));
  take(L.linear_out, size_t(kMaxRows) * m.max_linear * sizeof(float));
  take(L.logits, size_t(kMaxRows) * m.vocab_stride * sizeof(float));
  if (head_partial) take(L.head_partial, head_partial * sizeof(float));
  take(L.normed, kMaxRows * m.normed_stride * T);
  take(L.fused, kMaxRows * m.max_fused * T);
  take(L.mixed, kMaxRows * m.max_mixed * T);
  take(L.gate_up, kMaxRows * m.max_gate_up * T);
  take(L.act, kMaxRows * m.max_ff * T);
  take(L.head_rows, kMaxRows * m.normed_stride * T);
  take(s.gather_index, kMaxRows * sizeof(int32_t));
  L.rotations.resize(m.rotations.size());
  for (size_t i = 0; i < m.rotations.size(); ++i) take(L.rotations[i], s.capacity * (m.rotations[i].dims / 2) * sizeof(float2));
  L.runs.resize(m.runs.size());
  for (size_t i = 0; i < m.runs.size(); ++i) {
    const auto& l = m.layers[m.runs[i].layer];
    auto& r = L.runs[i];
    if (l.spec.mixer == EI_MIXER_MIN_GRU) {
      take(r.state, size_t(l.width_pad) * sizeof(float));
      take(r.ring_gate, size_t(kRingRows) * l.width_pad * sizeof(float));
      take(r.ring_candidate, size_t(kRingRows) * l.width_pad * sizeof(float));
    } else {
      take(r.k_cache, L.token_rows * l.spec.kv_heads * l.dim_pad * T);
      take(r.v_cache, L.token_rows * l.spec.kv_heads * l.vdim_pad * T);
      take(r.ring_k, size_t(kRingRows) * l.spec.lin_heads * l.lin_dim_pad * T);
      take(r.ring_v, size_t(kRingRows) * l.linear_width * T);
      take(r.state, size_t(l.linear_width) * l.lin_dim_pad * sizeof(float));
    }
  }
  EI_CUDA(cudaMalloc(reinterpret_cast<void**>(&s.arena), total));
  for (const auto& w : wanted) {
    void* at = s.arena + w.second;
    std::memcpy(w.first, &at, sizeof(at));
  }
  EI_CUDA(cudaMemset(s.arena, 0, total));
  for (size_t i = 0; i < m.rotations.size(); ++i)
    launch_rotation_table(L.rotations[i], s.capacity, m.rotations[i].dims, m.rotations[i].base, nullptr);
  EI_CUDA(cudaStreamSynchronize(nullptr));
}

void ensure_layered_workspace(ei_model& model) {
  auto& ws = model.prompt;
  if (ws.arena) return;
  LayeredModel& m = *model.layered;
  const size_t rows = std::min<size_t>(kPromptSegment, model.config.max_position_embeddings);
  const size_t chunks = (rows + kLightningChunk - 1) / kLightningChunk;
  std::vector<std::pair<void**, size_t>> wanted;
  size_t total = 0;
  auto take = [&](auto*& pointer, size_t bytes) {
    wanted.emplace_back(reinterpret_cast<void**>(&pointer), total);
    total += aligned(std::max<size_t>(bytes, 1));
  };
  const size_t partial_bytes = std::max(rows, size_t(16) * std::min<size_t>(rows, 256)) * m.residual_stride * sizeof(float);
  take(m.residual, rows * m.residual_stride * sizeof(float));
  take(m.linear_out, rows * m.max_linear * sizeof(float));
  take(m.chunk_states, chunks * m.max_chunk_state * sizeof(float));
  take(m.stretches, ((rows + kMinGruStretch - 1) / kMinGruStretch + 1) * 2 * m.max_rnn * sizeof(float));
  take(ws.normed, rows * m.normed_stride * 2);
  take(ws.qkv, rows * m.max_fused * 2);
  take(ws.attention, rows * m.max_mixed * 2);
  take(ws.gate_up, rows * m.max_gate_up * 2);
  take(ws.act, rows * m.max_ff * 2);
  take(ws.tokens, rows * 4);
  take(ws.step_tokens, rows * 4);
  take(ws.partial, partial_bytes);
  unsigned char* base = nullptr;
  EI_CUDA(cudaMalloc(reinterpret_cast<void**>(&base), total));
  if (cudaMemset(base, 0, total) != cudaSuccess || cudaStreamSynchronize(nullptr) != cudaSuccess ||
      cudaMallocHost(reinterpret_cast<void**>(&ws.host_tokens), rows * 4) != cudaSuccess) {
    cudaFree(base);
    throw std::runtime_error("Prompt workspace could not be set up");
  }
  for (const auto& w : wanted) {
    void* at = base + w.second;
    std::memcpy(w.first, &at, sizeof(at));
  }
  ws.partial_bytes = partial_bytes;
  ws.rows = rows;
  ws.arena = base;
}

void enqueue_layered_step(ei_session& s, int rows, StepKind kind) {
  if (s.model->layered->true32)
    enqueue_step_as<float>(s, rows, kind);
  else
    enqueue_step_as<bf16>(s, rows, kind);
}

void enqueue_layered_segment(ei_session& s, int rows) {
  ei_model& model = *s.model;
  const LayeredModel& m = *model.layered;
  LayeredSession& L = *s.layered;
  auto& ws = model.prompt;
  const bool pdl = true;
  const Buffers b{rows, ws.step_tokens, m.residual, m.linear_out, ws.normed, ws.qkv, ws.attention, ws.gate_up, ws.act};
  EmbedParams token{};
  token.tokens = ws.tokens;
  token.control = s.control;
  token.step_tokens = ws.step_tokens;
  token.vocab = int(model.config.vocab_size);
  token.rows = rows;
  token.capacity = int(s.capacity);
  enqueue_embed<bf16>(s, b, token);

  const auto sums = [&](const PreparedLinear& w, const bf16* x) {
    const int ksplit = prompt_gemm_ksplit(rows, w.out, w.in, model.multiprocessors, ws.partial_bytes);
    run_prompt_linear(s, w, x, rows, nullptr, pdl, ksplit);
    return ksplit;
  };
  for (size_t run = 0; run < m.runs.size(); ++run) {
    const LayeredModel::Layer& l = m.layers[m.runs[run].layer];
    const LayeredSession::Run& r = L.runs[run];
    run_prompt_linear_store(s, l.in, ws.normed, rows, ws.qkv, pdl);
    if (l.spec.mixer == EI_MIXER_MIN_GRU) {
      tick(s);
      tick(s);
      launch_min_gru_prompt(min_gru_params<bf16>(s, l, r, b), s.stream, pdl);
    } else {
      tick(s);
      launch_mixer_prepare<bf16>(prepare_params(s, l, r, b, false), s.stream, pdl);
      const SizedAttentionParams a = attention_params(s, l, r, b);
      tick(s);
      launch_sized_attention_prompt(a, s.stream, pdl);
      tick(s);
      int more = 0;
      launch_lightning_prompt(lightning_params<bf16>(s, l, r, b), s.stream, pdl, &more);
      s.launches += size_t(more - 1);
      tick(s);
      launch_mixer_finish<bf16>(finish_params<bf16>(s, l, b, a, false), s.stream, pdl);
    }
    int ksplit = sums(l.out, ws.attention);
    SublayerJoinParams j = join_params(s, b, ws.partial, ksplit);
    j.after = l.norm1b;
    if (l.spec.mlp == EI_MLP_NONE)
      end_of_run(s, b, run, j);
    else
      j.before = l.norm2;
    tick(s);
    launch_sublayer_join<bf16>(j, s.stream, pdl);
    if (l.spec.mlp == EI_MLP_NONE) continue;
    run_prompt_linear(s, l.gate_up, ws.normed, rows, ws.gate_up, pdl);
    tick(s);
    launch_clamped_glu<bf16>(ws.gate_up, rows, l.ff_pad, l.gate_up.glu_limit, ws.act, model.multiprocessors, s.stream, pdl);
    ksplit = sums(l.down, ws.act);
    j = join_params(s, b, ws.partial, ksplit);
    j.after = l.norm2b;
    end_of_run(s, b, run, j);
    tick(s);
    launch_sublayer_join<bf16>(j, s.stream, pdl);
  }
  enqueue_commit(s, rows, true);
}

void enqueue_layered_head(ei_session& s, const int32_t* device_rows, int count, bool greedy) {
  LayeredSession& L = *s.layered;
  bf16* rows = static_cast<bf16*>(L.head_rows);
  tick(s);
  launch_gather_rows<bf16>(s.model->prompt.normed, device_rows, count, s.model->layered->normed_stride, rows, s.stream);
  int parts = 0;
  run_head<bf16>(s, rows, count, greedy ? &parts : nullptr);
  if (!greedy) return;
  tick(s);
  launch_finalize(s.best_value, s.best_index, parts, count, s.targets, nullptr, nullptr, nullptr, nullptr, nullptr,
                  s.stream, true);
}

}  // namespace ei
