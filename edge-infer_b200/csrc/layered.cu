// Decoders described layer by layer: weights, caches and state, and the two forms of a forward.
//
// A step (at most 16 rows: decode, verify, a short portion) runs per layer, with programmatic dependent launch:
//   parallel mixer   fused projection -> heads prepared, K / V appended -> split attention -> linear attention step ->
//                    merge + gate -> output projection (FP32 sums)
//   gated recurrence fused projection -> recurrence step -> output projection (FP32 sums)
//   latent attention fused projection -> cache row, queries through the key expansion -> split attention -> merge, value
//                    expansion, gate -> output projection (FP32 sums)
//   state space,     fused projection (-> second factors of the low-rank ones) -> convolution and decays -> recurrence
//   channel delta    step -> norm and gate -> output projection (FP32 sums)
//   feed-forward     up (gate|up) with the activation in the epilogue -> down (FP32 sums)
// A sandwich block ends both sublayers with a join, which finishes one (norm after, residual add, what a loop pass adds)
// and starts the next (norm before); a parallel block has one join behind both. A prompt segment runs the same sequence
// over all its rows on the prompt GEMM, whole-history attention and the chunked forms of the recurrences. A model in true
// 32-bit runs every token through the step form.
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
  // A vector's values as FP32 on the host (zeros while only sizes are added up).
  std::vector<float> values(const std::string& name, size_t width) {
    const ei_named_tensor& t = find(name, width, 0);
    return base ? read(t) : std::vector<float>(width);
  }
  // The same spread over `heads` heads `pad` entries apart, on the device.
  const float* head_values(const std::string& name, int heads, int size, int pad) {
    const std::vector<float> from = values(name, size_t(heads) * size);
    std::vector<float> to(size_t(heads) * pad, 0.0f);
    for (int h = 0; h < heads; ++h) std::copy_n(from.begin() + size_t(h) * size, size, to.begin() + size_t(h) * pad);
    return host_values(to);
  }
  // Values `first`.. of a vector as `heads` heads `pad` entries apart from entry `at` on of `to`.
  static void spread(std::vector<float>& to, size_t at, const std::vector<float>& from, size_t first, int heads, int size, int pad) {
    for (int h = 0; h < heads; ++h)
      std::copy_n(from.begin() + first + size_t(h) * size, size, to.begin() + at + size_t(h) * pad);
  }
  // Rows `first`.. of a [channels, taps] convolution to the same places of every tap of [taps][channels].
  void conv_of(std::vector<float>& to, size_t channels, size_t at, const std::string& name, size_t rows, size_t first, int heads,
               int size, int pad, int taps) {
    const ei_named_tensor& t = find(name, rows, taps);
    if (!base) return;
    std::vector<uint16_t> bits(rows * taps);
    EI_CUDA(cudaMemcpy(bits.data(), t.data, bits.size() * 2, cudaMemcpyDefault));
    for (int h = 0; h < heads; ++h)
      for (int i = 0; i < size; ++i)
        for (int tap = 0; tap < taps; ++tap) {
          const uint32_t wide = uint32_t(bits[(first + size_t(h) * size + i) * taps + tap]) << 16;
          std::memcpy(&to[size_t(tap) * channels + at + size_t(h) * pad + i], &wide, 4);
        }
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
  // Output rows of `heads` heads of `size` features, `pad` rows apart; returns the row behind them. A head's rows may be
  // part of `spacing` rows in the source, from row `first` of a tensor of `total` rows on.
  int rows_of(bf16* weights, int pitch, int row, const std::string& name, int heads, int size, int pad, size_t inputs) {
    return some_rows_of(weights, pitch, row, name, size_t(heads) * size, 0, heads, size, size, pad, inputs);
  }
  int some_rows_of(bf16* weights, int pitch, int row, const std::string& name, size_t total, size_t first, int heads, int size,
                   int spacing, int pad, size_t inputs) {
    const ei_named_tensor& t = find(name, total, inputs);
    if (base)
      for (int h = 0; h < heads; ++h)
        copy(weights + (size_t(row) + size_t(h) * pad) * pitch, pitch,
             static_cast<const bf16*>(t.data) + (first + size_t(h) * spacing) * inputs, inputs, size, inputs);
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
  } else if (l.mixer == EI_MIXER_LATENT_ATTENTION) {
    if (!in_range(l.heads, 4096) || !in_range(l.dim, kMaxHeadDim) || !in_range(l.rot_dim, kMaxHeadDim) ||
        !in_range(l.vdim, kMaxHeadDim) || !in_range(l.kv_rank, kMaxLatent) || l.rot_dims > l.rot_dim || l.rot_dims % 2 ||
        !(l.rot_base > 0.0) || !std::isfinite(l.scale))
      throw std::invalid_argument("Layered decoder: invalid latent attention sizes (head sizes up to 512, latents up to 1024)");
    if (l.rot_factor != 0.0 && (!(l.rot_factor > 0.0) || !(l.rot_original > 0.0) || !(l.rot_fast > 0.0) || !(l.rot_slow > 0.0) ||
                                l.rot_base == 1.0 || !std::isfinite(l.rot_factor)))
      throw std::invalid_argument("Layered decoder: invalid rotation scaling");
  } else if (l.mixer == EI_MIXER_STATE_SPACE) {
    if (!in_range(l.heads, 4096) || !in_range(l.groups, 4096) || l.heads % l.groups || !in_range(l.state, kMaxHeadDim) ||
        !in_range(l.vdim, kMaxHeadDim) || !in_range(l.taps, 1024) || !in_range(l.norm_groups, kMany) ||
        (l.heads * l.vdim) % l.norm_groups)
      throw std::invalid_argument("Layered decoder: invalid state-space sizes (head sizes are limited to 512)");
  } else if (l.mixer == EI_MIXER_CHANNEL_DELTA) {
    if (!in_range(l.heads, 4096) || !in_range(l.kv_heads, 4096) || l.heads % l.kv_heads || !in_range(l.dim, kMaxHeadDim) ||
        !in_range(l.vdim, kMaxHeadDim) || !in_range(l.taps, 1024) || !in_range(l.decay_rank, kMany) || !in_range(l.gate_rank, kMany))
      throw std::invalid_argument("Layered decoder: invalid delta rule sizes (head sizes are limited to 512)");
  } else {
    throw std::invalid_argument("Layered decoder: unknown mixer");
  }
  const bool known = l.mlp == EI_MLP_NONE || l.mlp == EI_MLP_RELU_SQUARED || (l.mlp == EI_MLP_CLAMPED_GLU && !std::isnan(l.limit));
  if (!known || (l.mlp != EI_MLP_NONE && !in_range(l.ff, kMany)))
    throw std::invalid_argument("Layered decoder: invalid feed-forward");
}

// The rotation table's entry for these constants; equal ones share it.
int rotation_of(LayeredModel& m, Placement& at, const ei_layer_spec& s) {
  LayeredModel::Rotation r;
  r.dims = int(s.rot_dims);
  r.base = s.rot_base;
  r.factor = s.rot_factor;
  if (r.factor != 0.0) {
    r.original = s.rot_original;
    r.fast = s.rot_fast;
    r.slow = s.rot_slow;
  }
  for (size_t i = 0; i < m.rotations.size(); ++i) {
    const auto& o = m.rotations[i];
    if (o.dims == r.dims && o.base == r.base && o.factor == r.factor && o.original == r.original && o.fast == r.fast && o.slow == r.slow)
      return int(i);
  }
  // YaRN: frequencies that turn more than `fast` times over the original length stay, those below `slow` turns are
  // divided by the factor, a ramp in between; lengths grow by 0.1 ln(factor) + 1.
  double low = 0.0, high = 0.0;
  if (r.factor != 0.0) {
    const auto pair_of = [&](double turns) {
      return r.dims * std::log(r.original / (2.0 * M_PI * turns)) / (2.0 * std::log(r.base));
    };
    low = std::max(std::floor(pair_of(r.fast)), 0.0);
    high = std::min(std::ceil(pair_of(r.slow)), double(r.dims - 1));
    r.length = 0.1 * std::log(r.factor) + 1.0;
  }
  std::vector<double> frequencies;
  for (int i = 0; i < r.dims / 2; ++i) {
    const double f = std::pow(r.base, -2.0 * i / r.dims);
    const double ramp = r.factor != 0.0 ? std::min(std::max((i - low) / std::max(high - low, 0.001), 0.0), 1.0) : 0.0;
    frequencies.push_back(ramp == 0.0 ? f : f / r.factor * ramp + f * (1.0 - ramp));
  }
  r.frequencies = at.host_values(frequencies);
  m.rotations.push_back(r);
  return int(m.rotations.size()) - 1;
}

void place_min_gru(LayeredModel::Layer& L, Placement& at, const std::string& mix, size_t W, int K, int R) {
  bf16* weights = nullptr;
  const int width = int(L.spec.rnn_width);
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
}

void place_parallel(LayeredModel& m, LayeredModel::Layer& L, Placement& at, const std::string& mix, size_t W, int K, int R,
                    const double* decay) {
  bf16* weights = nullptr;
  const ei_layer_spec& s = L.spec;
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
  L.sink = at.host_values(at.values(left + "sink", H));
  bf16* norm = at.reserve<bf16>(L.linear_width);
  at.copy(norm, L.lin_vdim_pad, at.find(right + "norm", size_t(N) * s.lin_vdim, 0).data, s.lin_vdim, N, s.lin_vdim);
  L.lin_norm = norm;
  std::vector<float> powers;
  for (int h = 0; h < N; ++h)
    for (int n = 0; n <= kLightningChunk; ++n) powers.push_back(float(std::pow(decay[h], n)));
  L.powers = at.host_values(powers);
  L.rotation = rotation_of(m, at, s);
}

// Fused projection: q heads (unrotated | rotated) | latent | rotated key | gate.
void place_latent(LayeredModel& m, LayeredModel::Layer& L, Placement& at, const std::string& mix, size_t W, int K, int R) {
  bf16* weights = nullptr;
  const ei_layer_spec& s = L.spec;
  const int H = int(s.heads), dim = int(s.dim), rot = int(s.rot_dim), vdim = int(s.vdim), rank = int(s.kv_rank);
  L.dim_pad = round_up(dim, 16);
  L.rot_pad = round_up(rot, 16);
  L.vdim_pad = round_up(vdim, 16);
  L.rank_pad = round_up(rank, 64);
  L.row_pad = round_up(L.rank_pad + L.rot_pad, 64);
  const int query = L.dim_pad + L.rot_pad;
  L.latent_at = H * query;
  L.gate_at = L.latent_at + L.rank_pad + L.rot_pad;
  L.in = at.linear(K, L.gate_at + H * L.vdim_pad, &weights);
  const size_t q_rows = size_t(H) * (dim + rot);
  at.some_rows_of(weights, K, 0, mix + "q", q_rows, 0, H, dim, dim + rot, query, W);
  at.some_rows_of(weights, K, L.dim_pad, mix + "q", q_rows, dim, H, rot, dim + rot, query, W);
  at.some_rows_of(weights, K, L.latent_at, mix + "dkv", size_t(rank) + rot, 0, 1, rank, rank, L.rank_pad, W);
  at.some_rows_of(weights, K, L.latent_at + L.rank_pad, mix + "dkv", size_t(rank) + rot, rank, 1, rot, rot, L.rot_pad, W);
  at.rows_of(weights, K, L.gate_at, mix + "g", H, vdim, L.vdim_pad, W);
  L.latent_norm = at.vector(mix + "dkv.norm", rank, L.rank_pad);
  L.expand = at.linear(L.rank_pad, H * (L.dim_pad + L.vdim_pad), &weights);
  const int row = at.rows_of(weights, L.rank_pad, 0, mix + "uk", H, dim, L.dim_pad, rank);
  at.rows_of(weights, L.rank_pad, row, mix + "uv", H, vdim, L.vdim_pad, rank);
  L.out = at.linear(round_up(size_t(H) * L.vdim_pad, 64), R, &weights);
  at.columns_of(weights, L.out.in, 0, mix + "o", H, vdim, L.vdim_pad, W);
  L.rotation = rotation_of(m, at, s);
}

std::vector<float> exponentials(std::vector<float> v) {
  for (float& x : v) x = float(std::exp(double(x)));
  return v;
}

// Fused projection of both matrix recurrences: q heads | k heads | v heads | gate or first factors | step. A
// state-space layer's C, B and x take the places of q, k and v.
void place_state_space(LayeredModel::Layer& L, Placement& at, const std::string& mix, size_t W, int K, int R) {
  bf16* weights = nullptr;
  const ei_layer_spec& s = L.spec;
  const int H = int(s.heads), G = L.key_heads = int(s.groups), state = int(s.state), vdim = int(s.vdim), taps = int(s.taps);
  L.dim_pad = round_up(state, 16);
  L.vdim_pad = round_up(vdim, 16);
  const int keys = G * L.dim_pad, values = H * L.vdim_pad;
  L.channels = 2 * keys + values;
  L.gate_at = L.channels;
  L.step_at = L.gate_at + values;
  L.in = at.linear(K, L.step_at + round_up(H, 16), &weights);
  // Rows of the checkpoint's projection: gate | x | B | C | step; its convolution covers x | B | C.
  const size_t inner = size_t(H) * vdim, pairs = size_t(G) * state, rows = 2 * inner + 2 * pairs + H;
  at.some_rows_of(weights, K, 0, mix + "in", rows, 2 * inner + pairs, G, state, state, L.dim_pad, W);
  at.some_rows_of(weights, K, keys, mix + "in", rows, 2 * inner, G, state, state, L.dim_pad, W);
  at.some_rows_of(weights, K, 2 * keys, mix + "in", rows, inner, H, vdim, vdim, L.vdim_pad, W);
  at.some_rows_of(weights, K, L.gate_at, mix + "in", rows, 0, H, vdim, vdim, L.vdim_pad, W);
  at.some_rows_of(weights, K, L.step_at, mix + "in", rows, 2 * inner + 2 * pairs, 1, H, H, H, W);
  std::vector<float> conv(size_t(taps) * L.channels, 0.0f), bias(L.channels, 0.0f);
  const size_t convolved = inner + 2 * pairs;
  at.conv_of(conv, L.channels, 0, mix + "conv", convolved, inner + pairs, G, state, L.dim_pad, taps);
  at.conv_of(conv, L.channels, keys, mix + "conv", convolved, inner, G, state, L.dim_pad, taps);
  at.conv_of(conv, L.channels, 2 * keys, mix + "conv", convolved, 0, H, vdim, L.vdim_pad, taps);
  L.conv = at.host_values(conv);
  const std::vector<float> given = at.values(mix + "conv.b", convolved);
  Placement::spread(bias, 0, given, inner + pairs, G, state, L.dim_pad);
  Placement::spread(bias, keys, given, inner, G, state, L.dim_pad);
  Placement::spread(bias, 2 * keys, given, 0, H, vdim, L.vdim_pad);
  L.conv_bias = at.host_values(bias);
  L.rate = at.host_values(exponentials(at.values(mix + "A_log", H)));
  L.bias = at.host_values(at.values(mix + "dt_bias", H));
  L.skip = at.host_values(at.values(mix + "D", H));
  bf16* norm = at.reserve<bf16>(values);
  at.copy(norm, L.vdim_pad, at.find(mix + "norm", inner, 0).data, vdim, H, vdim);
  L.state_norm = norm;
  L.out = at.linear(round_up(values, 64), R, &weights);
  at.columns_of(weights, L.out.in, 0, mix + "o", H, vdim, L.vdim_pad, W);
}

void place_channel_delta(LayeredModel::Layer& L, Placement& at, const std::string& mix, size_t W, int K, int R) {
  bf16* weights = nullptr;
  const ei_layer_spec& s = L.spec;
  const int H = int(s.heads), G = L.key_heads = int(s.kv_heads), dim = int(s.dim), vdim = int(s.vdim), taps = int(s.taps);
  const int decay = int(s.decay_rank), gate = int(s.gate_rank);
  L.dim_pad = round_up(dim, 16);
  L.vdim_pad = round_up(vdim, 16);
  const int keys = G * L.dim_pad, values = H * L.vdim_pad, decay_pad = round_up(decay, 64), gate_pad = round_up(gate, 64);
  L.channels = 2 * keys + values;
  L.first_at = L.channels;
  L.step_at = L.first_at + decay_pad + gate_pad;
  L.in = at.linear(K, L.step_at + round_up(H, 16), &weights);
  at.rows_of(weights, K, 0, mix + "q", G, dim, L.dim_pad, W);
  at.rows_of(weights, K, keys, mix + "k", G, dim, L.dim_pad, W);
  at.rows_of(weights, K, 2 * keys, mix + "v", H, vdim, L.vdim_pad, W);
  at.rows_of(weights, K, L.first_at, mix + "a1", 1, decay, decay_pad, W);
  at.rows_of(weights, K, L.first_at + decay_pad, mix + "g1", 1, gate, gate_pad, W);
  at.rows_of(weights, K, L.step_at, mix + "b", 1, H, H, W);
  // Both second factors in one projection of both first factors' results: two blocks on the diagonal.
  L.gate_at = H * L.dim_pad;
  L.second = at.linear(decay_pad + gate_pad, H * L.dim_pad + values, &weights);
  at.rows_of(weights, L.second.in, 0, mix + "a2", H, dim, L.dim_pad, decay);
  at.rows_of(weights + decay_pad, L.second.in, L.gate_at, mix + "g2", H, vdim, L.vdim_pad, gate);
  std::vector<float> conv(size_t(taps) * L.channels, 0.0f);
  at.conv_of(conv, L.channels, 0, mix + "q.conv", size_t(G) * dim, 0, G, dim, L.dim_pad, taps);
  at.conv_of(conv, L.channels, keys, mix + "k.conv", size_t(G) * dim, 0, G, dim, L.dim_pad, taps);
  at.conv_of(conv, L.channels, 2 * keys, mix + "v.conv", size_t(H) * vdim, 0, H, vdim, L.vdim_pad, taps);
  L.conv = at.host_values(conv);
  L.rate = at.host_values(exponentials(at.values(mix + "A_log", H)));
  L.bias = at.head_values(mix + "dt_bias", H, dim, L.dim_pad);
  bf16* norm = at.reserve<bf16>(values);
  const ei_named_tensor& shared = at.find(mix + "norm", vdim, 0);
  for (int h = 0; h < H; ++h) at.copy(norm + size_t(h) * L.vdim_pad, vdim, shared.data, vdim, 1, vdim);
  L.state_norm = norm;
  L.out = at.linear(round_up(values, 64), R, &weights);
  at.columns_of(weights, L.out.in, 0, mix + "o", H, vdim, L.vdim_pad, W);
}

void place(ei_model& model, const ei_layered_config& c, const ei_layer_spec* specs, Placement& at) {
  LayeredModel& m = *model.layered;
  const size_t W = c.width, V = c.vocab_size;
  const int R = m.residual_stride, K = m.normed_stride;
  at.offset = 0;
  m.layers.assign(c.n_layers, {});
  m.rotations.clear();
  bf16* weights = nullptr;
  m.head = at.linear(K, m.vocab_stride, &weights);
  if (c.tied_head) {
    at.rows_of(weights, K, 0, "embed", 1, int(V), int(V), W);
    m.embedding = weights;
    m.embedding_stride = K;
  } else {
    at.rows_of(weights, K, 0, "head", 1, int(V), int(V), W);
    m.embedding = at.matrix("embed", V, W, V, R);
    m.embedding_stride = R;
  }
  if (c.pair_buckets) {
    m.pairs.table = at.matrix("bigram", c.pair_buckets + 1, W, c.pair_buckets + 1, R);
    m.pairs.stride = R;
    m.pairs.buckets = c.pair_buckets;
    m.pairs.mul_prev = c.pair_mul_prev % c.pair_buckets;
    m.pairs.mul_cur = c.pair_mul_cur % c.pair_buckets;
  }
  if (c.loop_times) m.loop_step = at.matrix("loop.step", c.loop_times, W, c.loop_times, R);
  if (m.parallel)
    m.final_weight = at.vector("final.norm", W, R);
  else
    m.final_norm = at.norm("final.norm", W, R);
  for (size_t i = 0; i < c.n_layers; ++i) {
    const std::string p = "l" + std::to_string(i) + ".", mix = p + "mix.";
    LayeredModel::Layer& L = m.layers[i];
    const ei_layer_spec& s = L.spec = specs[i];
    L.spec.decay = nullptr;
    const bool feeds = s.mlp != EI_MLP_NONE;
    if (m.parallel) {
      L.norm1_weight = at.vector(p + "norm1", W, R);
      L.scale1 = at.vector(p + "ls1", W, R);
      if (feeds) {
        L.norm2_weight = at.vector(p + "norm2", W, R);
        L.scale2 = at.vector(p + "ls2", W, R);
      }
    } else {
      L.norm1 = at.norm(p + "norm1", W, R);
      L.norm1b = at.norm(p + "norm1b", W, R);
      if (feeds) {
        L.norm2 = at.norm(p + "norm2", W, R);
        L.norm2b = at.norm(p + "norm2b", W, R);
      }
    }
    switch (s.mixer) {
      case EI_MIXER_MIN_GRU: place_min_gru(L, at, mix, W, K, R); break;
      case EI_MIXER_PARALLEL: place_parallel(m, L, at, mix, W, K, R, specs[i].decay); break;
      case EI_MIXER_LATENT_ATTENTION: place_latent(m, L, at, mix, W, K, R); break;
      case EI_MIXER_STATE_SPACE: place_state_space(L, at, mix, W, K, R); break;
      default: place_channel_delta(L, at, mix, W, K, R); break;
    }
    if (L.outer()) {
      L.raw_rows = 1;  // a step reads the taps behind its first row while it records its own rows
      while (L.raw_rows < kPendingRows + int(s.taps) - 1) L.raw_rows *= 2;
    }
    if (!feeds) continue;
    L.ff_pad = round_up(s.ff, 64);
    if (s.mlp == EI_MLP_RELU_SQUARED) {
      L.up = at.linear(K, L.ff_pad, &weights);
      L.up.activation = kActReluSquared;
      at.rows_of(weights, K, 0, p + "mlp.up", 1, int(s.ff), L.ff_pad, W);
    } else {
      L.gate_up = at.linear(K, 2 * L.ff_pad, &weights);
      L.gate_up.glu = kGluClamped;
      L.gate_up.glu_limit = float(s.limit);
      at.rows_of(weights, K, 0, p + "mlp.gate", 1, int(s.ff), L.ff_pad, W);
      at.rows_of(weights, K, L.ff_pad, p + "mlp.up", 1, int(s.ff), L.ff_pad, W);
    }
    L.down = at.linear(L.ff_pad, R, &weights);
    at.columns_of(weights, L.ff_pad, 0, p + "mlp.down", 1, int(s.ff), L.ff_pad, W);
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
  static int sums(ei_session& s, const PreparedLinear& w, const bf16* x, int rows, int x_stride = 0) {
    int ksplit = 1;
    run_linear(s, w, x, rows, kEpiPartial, nullptr, 0, true, &ksplit, x_stride);
    return ksplit;
  }
  static void store(ei_session& s, const PreparedLinear& w, const bf16* x, int rows, bf16* out, int x_stride = 0) {
    if (has_plan(s, w, rows, kEpiStore)) {
      run_linear(s, w, x, rows, kEpiStore, out, w.out, true, nullptr, x_stride);
      return;
    }
    const int ksplit = sums(s, w, x, rows, x_stride);
    tick(s);
    launch(splitk_store_kernel, dim3(std::min(s.model->multiprocessors * 8, (rows * w.out + 255) / 256)), dim3(256), 0,
           s.stream, true, (const float*)s.partial, ksplit, rows, w.out, w.bias, out, w.out, w.activation);
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
  static int sums(ei_session& s, const PreparedLinear& w, const float* x, int rows, int x_stride = 0) {
    store(s, w, x, rows, s.partial, x_stride);
    return 1;
  }
  static void store(ei_session& s, const PreparedLinear& w, const float* x, int rows, float* out, int x_stride = 0) {
    tick(s);
    launch_true32_linear(x, x_stride ? x_stride : w.in, rows, w, out, s.stream, true);
  }
  static void gated(ei_session& s, const PreparedLinear& w, const float* x, int rows, float* pair, float* out) {
    store(s, w, x, rows, pair);
    tick(s);
    launch_clamped_glu<float>(pair, rows, w.out / 2, w.glu_limit, out, s.model->multiprocessors, s.stream, true);
  }
};

// FP32 sums of a step projection in a buffer other than the session's.
template <typename T>
int sums_into(ei_session& s, const PreparedLinear& w, const T* x, int rows, float* buffer) {
  struct Lend {
    ei_session& s;
    float* keep;
    ~Lend() { s.partial = keep; }
  } lend{s, s.partial};
  s.partial = buffer;
  return StepLinear<T>::sums(s, w, x, rows);
}

// The vocabulary head over at most 16 rows: FP32 logits in the session; with `parts` the argmax partials too.
template <typename T>
void run_head(ei_session& s, const T* rows_in, int rows, int* parts) {
  const LayeredModel& m = *s.model->layered;
  LayeredSession& L = *s.layered;
  const int ksplit = sums_into<T>(s, m.head, rows_in, rows, L.head_partial ? L.head_partial : L.logits);
  if (L.head_partial || m.softcap > 0.0f) {
    tick(s);
    launch_sum_partials(L.head_partial ? L.head_partial : L.logits, ksplit, size_t(rows) * m.vocab_stride, m.softcap, L.logits,
                        s.model->multiprocessors, s.stream, true);
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
  void *second_normed, *second;  // a parallel block's other norm; second factors of a low-rank projection
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

// The norms that open layer run `run` of a parallel model, or the final one.
RowNorms row_norms(const LayeredModel& m, const Buffers& b, size_t run) {
  RowNorms n;
  n.width = m.width;
  n.stride = m.normed_stride;
  n.eps = m.eps;
  n.normed_first = b.normed;
  n.first = m.final_weight;
  if (run < m.runs.size()) {
    const auto& l = m.layers[m.runs[run].layer];
    n.first = l.norm1_weight;
    n.second = l.norm2_weight;
    n.normed_second = b.second_normed;
  }
  return n;
}

template <typename T>
void enqueue_embed(ei_session& s, const Buffers& b, const EmbedParams& token) {
  const LayeredModel& m = *s.model->layered;
  tick(s);
  if (m.parallel) {
    ParallelEmbedParams e{};
    e.token = token;
    e.table = m.embedding;
    e.table_stride = m.embedding_stride;
    e.pairs = m.pairs;
    e.pairs.history = s.layered->history;
    e.residual = b.residual;
    e.residual_stride = m.residual_stride;
    e.norms = row_norms(m, b, 0);
    launch_parallel_embed<T>(e, s.stream, false);
    return;
  }
  LayeredEmbedParams e{};
  e.token = token;
  e.table = m.embedding;
  if (m.runs[0].pass >= 0) e.vector = m.loop_step + size_t(m.runs[0].pass) * m.residual_stride;
  e.norm = norm_ahead(m, 0);
  e.residual = b.residual;
  e.residual_stride = m.residual_stride;
  e.normed = b.normed;
  e.normed_stride = m.normed_stride;
  launch_layered_embed<T>(e, s.stream, false);
}

// The join that ends layer run `run` of a parallel model.
template <typename T>
void enqueue_parallel_join(ei_session& s, const Buffers& b, size_t run, const float* mixed, int mixed_ksplit, const float* fed,
                           int fed_ksplit) {
  const LayeredModel& m = *s.model->layered;
  const LayeredSession& L = *s.layered;
  const auto& l = m.layers[m.runs[run].layer];
  ParallelJoinParams j{};
  j.mixed = mixed;
  j.mixed_ksplit = mixed_ksplit;
  j.fed = fed;
  j.fed_ksplit = fed_ksplit;
  j.rows = b.rows;
  j.mixed_scale = l.scale1;
  j.fed_scale = l.scale2;
  j.residual = b.residual;
  j.residual_stride = m.residual_stride;
  if (L.tap) {
    j.tap = L.tap + run * L.tap_rows * m.width;
    j.tap_width = m.width;
  }
  j.norms = row_norms(m, b, run + 1);
  tick(s);
  launch_parallel_join<T>(j, s.stream, true);
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
  a.k_stride = int(l.spec.kv_heads) * l.dim_pad;
  a.v_stride = int(l.spec.kv_heads) * l.vdim_pad;
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

LatentParams latent_params(const ei_session& s, const LayeredModel::Layer& l, const LayeredSession::Run& r, const Buffers& b) {
  LatentParams p{};
  p.fused = b.fused;
  p.rows = b.rows;
  p.stride = l.in.out;
  p.latent_at = l.latent_at;
  p.gate_at = l.gate_at;
  p.heads = int(l.spec.heads);
  p.dim_pad = l.dim_pad;
  p.vdim_pad = l.vdim_pad;
  p.rank = int(l.spec.kv_rank);
  p.rank_pad = l.rank_pad;
  p.rot_pad = l.rot_pad;
  p.rot_dims = int(l.spec.rot_dims);
  p.row_pad = l.row_pad;
  p.eps = s.model->layered->eps;
  p.norm = l.latent_norm;
  p.rotation = s.layered->rotations[l.rotation];
  p.expand = l.expand.dense;
  p.cache = r.latent;
  p.control = s.control;
  p.capacity = int(s.capacity);
  p.query = s.layered->latent_query;
  p.out = b.mixed;
  p.out_stride = l.out.in;
  return p;
}

// Attention of a step's queries over the latent cache; partials in the session's scratch, or (plain form) finished
// latents in `out`.
SizedAttentionParams latent_scores(ei_session& s, const LayeredModel::Layer& l, const LayeredSession::Run& r, const Buffers& b) {
  SizedAttentionParams a{};
  a.q = s.layered->latent_query;
  a.q_stride = int(l.spec.heads) * l.row_pad;
  a.k = a.v = r.latent;
  a.k_stride = a.v_stride = l.row_pad;
  a.rows = b.rows;
  a.heads = int(l.spec.heads);
  a.kv_heads = 1;
  a.dim_pad = l.row_pad;
  a.vdim_pad = l.rank_pad;
  a.scale = float(l.spec.scale);
  a.out_scale = 1.0f;
  a.device_offset = &s.control->context;
  a.capacity = int(s.capacity);
  a.chunk = s.attention_chunk;
  a.max_splits = s.attention_splits;
  a.scratch = s.attention_scratch;
  a.out = s.layered->latent_out;
  a.out_stride = int(l.spec.heads) * l.rank_pad;
  a.status = &s.control->status;
  if (s.inject_attention_polls) {
    a.wait_limit = s.inject_attention_polls;
    a.fault_tx = 16;
    s.inject_attention_polls = 0;  // one launch only
  }
  return a;
}

OuterStateParams outer_params(const ei_session& s, const LayeredModel::Layer& l, const LayeredSession::Run& r, const Buffers& b) {
  OuterStateParams p{};
  p.delta = l.delta();
  p.fused = b.fused;
  p.rows = b.rows;
  p.stride = l.in.out;
  p.step_at = l.step_at;
  p.heads = int(l.spec.heads);
  p.key_heads = l.key_heads;
  p.dim = int(l.delta() ? l.spec.dim : l.spec.state);
  p.dim_pad = l.dim_pad;
  p.vdim = int(l.spec.vdim);
  p.vdim_pad = l.vdim_pad;
  p.taps = int(l.spec.taps);
  p.conv = l.conv;
  p.conv_bias = l.conv_bias;
  p.raw = r.raw;
  p.raw_rows = l.raw_rows;
  p.decay = b.second;
  p.decay_stride = l.second.out;
  p.rate = l.rate;
  p.bias = l.bias;
  p.skip = l.skip;
  p.ring_k = r.ring_key;
  p.ring_g = r.ring_decay;
  p.ring_u = r.ring_write;
  p.q = s.layered->state_q;
  p.v = s.layered->state_v;
  p.beta = s.layered->state_beta;
  p.state = r.state;
  p.control = s.control;
  p.capacity = int(s.capacity);
  p.out = b.linear_out;
  return p;
}

template <typename T>
StateFinishParams state_finish_params(const ei_session& s, const LayeredModel::Layer& l, const Buffers& b) {
  StateFinishParams f{};
  f.in = b.linear_out;
  f.rows = b.rows;
  f.heads = int(l.spec.heads);
  f.vdim = int(l.spec.vdim);
  f.vdim_pad = l.vdim_pad;
  f.gate_first = !l.delta();
  f.groups = int(l.delta() ? l.spec.heads : l.spec.norm_groups);
  f.gate = static_cast<const T*>(l.delta() ? b.second : b.fused) + l.gate_at;
  f.gate_stride = l.delta() ? l.second.out : l.in.out;
  f.norm = l.state_norm;
  f.eps = s.model->layered->eps;
  f.out = b.mixed;
  f.out_stride = l.out.in;
  return f;
}

// A layer's token mixer from the normed rows to the activations of its output projection, at most 16 rows.
template <typename T>
void enqueue_mixer_step(ei_session& s, const LayeredModel::Layer& l, const LayeredSession::Run& r, const Buffers& b) {
  const ei_model& model = *s.model;
  const bool pdl = true, true32 = model.layered->true32;
  StepLinear<T>::store(s, l.in, static_cast<const T*>(b.normed), b.rows, static_cast<T*>(b.fused));
  switch (l.spec.mixer) {
    case EI_MIXER_MIN_GRU:
      tick(s);
      launch_min_gru_step<T>(min_gru_params<T>(s, l, r, b), s.stream, pdl);
      return;
    case EI_MIXER_PARALLEL: {
      tick(s);
      launch_mixer_prepare<T>(prepare_params(s, l, r, b, true), s.stream, pdl);
      const SizedAttentionParams a = attention_params(s, l, r, b);
      const bool tiled = !true32 && sized_attention_ok(l.dim_pad, l.vdim_pad);
      tick(s);
      if (tiled)
        launch_sized_attention_step(a, s.stream, pdl);
      else
        launch_plain_attention<T>(a, s.stream, pdl);
      tick(s);
      launch_lightning_step<T>(lightning_params<T>(s, l, r, b), s.stream, pdl);
      tick(s);
      launch_mixer_finish<T>(finish_params<T>(s, l, b, a, tiled), s.stream, pdl);
      return;
    }
    case EI_MIXER_LATENT_ATTENTION: {
      const LatentParams p = latent_params(s, l, r, b);
      const bool tiled = !true32 && latent_attention_ok(l.rank_pad, l.row_pad, model.smem_limit);
      tick(s);
      launch_latent_prepare<T>(p, true, s.stream, pdl);
      const SizedAttentionParams a = latent_scores(s, l, r, b);
      tick(s);
      if (tiled)
        launch_latent_attention(a, l.row_pad, model.smem_limit, s.stream, pdl);
      else
        launch_plain_attention<T>(a, s.stream, pdl);
      tick(s);
      launch_latent_expand<T>(p, a, tiled, s.stream, pdl);
      return;
    }
    default: {
      if (l.delta())
        StepLinear<T>::store(s, l.second, static_cast<const T*>(b.fused) + l.first_at, b.rows, static_cast<T*>(b.second), l.in.out);
      const OuterStateParams p = outer_params(s, l, r, b);
      tick(s);
      launch_outer_prepare<T>(p, s.stream, pdl);
      tick(s);
      launch_outer_step(p, s.stream, pdl);
      tick(s);
      launch_state_finish<T>(state_finish_params<T>(s, l, b), s.stream, pdl);
      return;
    }
  }
}

template <typename T>
void enqueue_step_as(ei_session& s, int rows, StepKind kind) {
  const LayeredModel& m = *s.model->layered;
  LayeredSession& L = *s.layered;
  const bool pdl = true;
  const size_t before = s.launches;
  const Buffers b{rows,    s.step_tokens, L.residual, L.linear_out,    L.normed, L.fused,
                  L.mixed, L.gate_up,     L.act,      L.second_normed, L.second};
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
    enqueue_mixer_step<T>(s, l, L.runs[run], b);
    const bool feeds = l.spec.mlp != EI_MLP_NONE;
    const T *normed = static_cast<const T*>(m.parallel ? b.second_normed : b.normed), *mixed = static_cast<const T*>(b.mixed);
    T* act = static_cast<T*>(b.act);
    const auto activate = [&] {
      if (l.spec.mlp == EI_MLP_RELU_SQUARED)
        StepLinear<T>::store(s, l.up, normed, rows, act);
      else
        StepLinear<T>::gated(s, l.gate_up, normed, rows, static_cast<T*>(b.gate_up), act);
    };
    if (m.parallel) {
      const int mixed_ksplit = sums_into<T>(s, l.out, mixed, rows, L.mixed_partial);
      int fed_ksplit = 0;
      if (feeds) {
        activate();
        fed_ksplit = StepLinear<T>::sums(s, l.down, act, rows);
      }
      enqueue_parallel_join<T>(s, b, run, L.mixed_partial, mixed_ksplit, feeds ? s.partial : nullptr, fed_ksplit);
      continue;
    }
    int ksplit = StepLinear<T>::sums(s, l.out, mixed, rows);
    SublayerJoinParams j = join_params(s, b, s.partial, ksplit);
    j.after = l.norm1b;
    if (feeds)
      j.before = l.norm2;
    else
      end_of_run(s, b, run, j);
    tick(s);
    launch_sublayer_join<T>(j, s.stream, pdl);
    if (!feeds) continue;
    activate();
    ksplit = StepLinear<T>::sums(s, l.down, act, rows);
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
  if (c.pair_buckets && !positive(c.pair_buckets, kMany)) throw std::invalid_argument("Layered decoder: pair table out of range");
  if (!std::isfinite(c.logit_softcap) || c.logit_softcap < 0.0) throw std::invalid_argument("Layered decoder: invalid logit cap");
  if (c.block != EI_BLOCK_SANDWICH && c.block != EI_BLOCK_PARALLEL) throw std::invalid_argument("Layered decoder: unknown block form");
  if (c.block == EI_BLOCK_PARALLEL ? c.loop_times != 0 : c.pair_buckets != 0)
    throw std::invalid_argument("Layered decoder: loops go with sandwich blocks, the pair table with parallel ones");
  for (size_t i = 0; i < c.n_layers; ++i) validate_layer(specs[i]);

  model.layered = std::make_shared<LayeredModel>();
  LayeredModel& m = *model.layered;
  m.true32 = c.true32 != 0;
  m.parallel = c.block == EI_BLOCK_PARALLEL;
  m.softcap = float(c.logit_softcap);
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
    model.weight_bytes += l.in.bytes + l.out.bytes + l.gate_up.bytes + l.up.bytes + l.down.bytes + l.expand.bytes + l.second.bytes;
  }
  model.prompt_ready = !m.true32;
  for (const auto& l : m.layers) {
    m.max_fused = std::max(m.max_fused, l.in.out);
    m.max_mixed = std::max(m.max_mixed, l.out.in);
    m.max_gate_up = std::max(m.max_gate_up, l.gate_up.out);
    m.max_ff = std::max(m.max_ff, l.ff_pad);
    m.max_linear = std::max(m.max_linear, l.outer() ? int(l.spec.heads) * l.vdim_pad : l.linear_width);
    m.max_rnn = std::max(m.max_rnn, l.width_pad);
    if (l.outer()) {
      m.max_second = std::max(m.max_second, l.second.out);
      m.max_state_keys = std::max(m.max_state_keys, l.key_heads * l.dim_pad);
      m.max_state_heads = std::max(m.max_state_heads, int(l.spec.heads));
      m.max_channels = std::max(m.max_channels, l.channels);
      if (l.delta()) {
        model.prompt_ready = model.prompt_ready && delta_prompt_ok(l.dim_pad, l.vdim_pad) && prompt_linear_ok(l.second);
        m.max_delta_chunks = std::max(m.max_delta_chunks, delta_prompt_bytes(kPromptSegment, l.spec.heads, l.dim_pad, l.vdim_pad));
      } else {
        model.prompt_ready = model.prompt_ready && lightning_prompt_ok(l.dim_pad, l.vdim_pad);
        m.max_chunk_state = std::max(m.max_chunk_state, size_t(l.spec.heads) * l.vdim_pad * l.dim_pad);
      }
    }
    if (l.spec.mixer == EI_MIXER_LATENT_ATTENTION) {
      m.max_expand = std::max(m.max_expand, size_t(l.expand.out));
      model.prompt_ready = model.prompt_ready && sized_attention_ok(l.dim_pad + l.rot_pad, l.vdim_pad) && prompt_linear_ok(l.expand);
    }
    if (l.spec.mixer == EI_MIXER_PARALLEL) {
      m.max_chunk_state = std::max(m.max_chunk_state, size_t(l.linear_width) * l.lin_dim_pad);
      model.prompt_ready = model.prompt_ready && sized_attention_ok(l.dim_pad, l.vdim_pad) &&
                           lightning_prompt_ok(l.lin_dim_pad, l.lin_vdim_pad);
    }
    const PreparedLinear& widen = l.spec.mlp == EI_MLP_RELU_SQUARED ? l.up : l.gate_up;
    model.prompt_ready = model.prompt_ready && prompt_linear_ok(l.in) && prompt_linear_ok(l.out) &&
                         (l.spec.mlp == EI_MLP_NONE || (prompt_linear_ok(widen) && prompt_linear_ok(l.down)));
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
  size_t partial = 0, scratch = 0, mixed_partial = 0, latent_query = 0, latent_out = 0;
  for (const auto& l : m.layers) {
    for (const PreparedLinear* w : {&l.in, &l.out, &l.gate_up, &l.up, &l.down, &l.second}) partial = std::max(partial, partial_floats(*w));
    if (m.parallel) mixed_partial = std::max(mixed_partial, partial_floats(l.out));
    if (l.spec.mixer == EI_MIXER_LATENT_ATTENTION) {
      scratch = std::max(scratch, sized_attention_scratch_bytes(kMaxRows, l.spec.heads, l.rank_pad, s.capacity));
      latent_query = std::max(latent_query, size_t(l.spec.heads) * l.row_pad);
      latent_out = std::max(latent_out, size_t(l.spec.heads) * l.rank_pad);
    }
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
  if (m.parallel) {
    take(L.mixed_partial, mixed_partial * sizeof(float));
    take(L.second_normed, kMaxRows * m.normed_stride * T);
  }
  if (m.pairs.table) take(L.history, s.capacity * sizeof(uint32_t));
  take(L.second, size_t(kMaxRows) * m.max_second * T);
  take(L.state_q, size_t(kMaxRows) * m.max_state_keys * sizeof(float));
  take(L.state_v, size_t(kMaxRows) * m.max_linear * sizeof(float));
  take(L.state_beta, size_t(kMaxRows) * m.max_state_heads * sizeof(float));
  take(L.latent_query, kMaxRows * latent_query * T);
  take(L.latent_out, kMaxRows * latent_out * T);
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
    } else if (l.spec.mixer == EI_MIXER_LATENT_ATTENTION) {
      take(r.latent, L.token_rows * l.row_pad * T);
    } else if (l.outer()) {
      const size_t heads = l.spec.heads;
      take(r.raw, size_t(l.raw_rows) * l.channels * T);
      take(r.ring_key, size_t(kRingRows) * l.key_heads * l.dim_pad * sizeof(float));
      take(r.ring_decay, size_t(kRingRows) * heads * (l.delta() ? l.dim_pad : 1) * sizeof(float));
      take(r.ring_write, size_t(kRingRows) * heads * l.vdim_pad * sizeof(float));
      take(r.state, heads * l.vdim_pad * l.dim_pad * sizeof(float));
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
    launch_rotation_table(L.rotations[i], s.capacity, m.rotations[i].frequencies, m.rotations[i].dims / 2, m.rotations[i].length, nullptr);
  EI_CUDA(cudaStreamSynchronize(nullptr));
}

void ensure_expanded(ei_model& model, size_t tokens) {
  LayeredModel& m = *model.layered;
  const size_t bytes = tokens * m.max_expand * sizeof(bf16);
  if (bytes <= m.expanded_bytes) return;
  if (m.expanded) EI_CUDA(cudaFree(m.expanded));
  m.expanded = nullptr;
  m.expanded_bytes = 0;
  const size_t room = bytes + bytes / 4;
  EI_CUDA(cudaMalloc(reinterpret_cast<void**>(&m.expanded), room));
  m.expanded_bytes = room;
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
  if (m.parallel) {
    take(m.mixed_partial, partial_bytes);
    take(m.second_normed, rows * m.normed_stride * 2);
  }
  if (m.max_channels) {
    take(m.second, rows * m.max_second * 2);
    take(m.conv_out, rows * m.max_channels * 2);
    take(m.inverse, rows * 2 * m.max_state_heads * sizeof(float));
    take(m.decay_totals, chunks * m.max_state_heads * sizeof(float));
    take(m.delta_chunks, m.max_delta_chunks);
  }
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

// A layer's token mixer over a prompt segment, from the normed rows to the activations of its output projection.
static void enqueue_mixer_segment(ei_session& s, const LayeredModel::Layer& l, const LayeredSession::Run& r, const Buffers& b, size_t context) {
  ei_model& model = *s.model;
  const LayeredModel& m = *model.layered;
  const bool pdl = true;
  const int rows = b.rows;
  run_prompt_linear_store(s, l.in, static_cast<const bf16*>(b.normed), rows, static_cast<bf16*>(b.fused), pdl);
  switch (l.spec.mixer) {
    case EI_MIXER_MIN_GRU:
      tick(s);
      tick(s);
      launch_min_gru_prompt(min_gru_params<bf16>(s, l, r, b), s.stream, pdl);
      return;
    case EI_MIXER_PARALLEL: {
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
      return;
    }
    case EI_MIXER_LATENT_ATTENTION: {
      const LatentParams p = latent_params(s, l, r, b);
      tick(s);
      launch_latent_prepare<bf16>(p, false, s.stream, pdl);
      // Keys and values of every token so far, from the cached latents.
      const int tokens = int(context) + rows, keys = p.heads * l.dim_pad;
      run_prompt_linear(s, l.expand, static_cast<const bf16*>(r.latent), tokens, m.expanded, pdl, 0, l.row_pad);
      SizedAttentionParams a{};
      a.q = b.fused;
      a.q_stride = l.in.out;
      a.k = m.expanded;
      a.v = m.expanded + keys;
      a.k_stride = a.v_stride = l.expand.out;
      a.rows = rows;
      a.heads = a.kv_heads = p.heads;
      a.dim_pad = l.dim_pad + l.rot_pad;
      a.vdim_pad = l.vdim_pad;
      a.shared = static_cast<const bf16*>(r.latent) + l.rank_pad;
      a.shared_stride = l.row_pad;
      a.shared_pad = l.rot_pad;
      a.tokens = tokens;
      a.fresh = true;
      a.gate = static_cast<const bf16*>(b.fused) + l.gate_at;
      a.gate_stride = l.in.out;
      a.scale = float(l.spec.scale);
      a.out_scale = 1.0f;
      a.device_offset = &s.control->context;
      a.capacity = int(s.capacity);
      a.out = b.mixed;
      a.out_stride = l.out.in;
      a.status = &s.control->status;
      if (s.inject_attention_polls) {
        a.wait_limit = s.inject_attention_polls;
        a.fault_tx = 16;
        s.inject_attention_polls = 0;  // one launch only
      }
      tick(s);
      launch_sized_attention_prompt(a, s.stream, pdl);
      return;
    }
    default: {
      const OuterStateParams p = outer_params(s, l, r, b);
      if (l.delta())
        run_prompt_linear(s, l.second, static_cast<const bf16*>(b.fused) + l.first_at, rows, static_cast<bf16*>(b.second), pdl, 0, l.in.out);
      tick(s);
      launch_outer_conv(p, m.conv_out, m.inverse, s.stream, pdl);
      const int keys = p.key_heads * p.dim_pad;
      if (l.delta()) {
        DeltaPromptParams d{};
        d.outer = p;
        d.conv = m.conv_out;
        d.inverse = m.inverse;
        d.channels = l.channels;
        d.chunks = m.delta_chunks;
        tick(s);
        tick(s);
        launch_delta_prompt(d, s.stream, pdl);
      } else {
        LightningParams q{};
        q.q = m.conv_out;
        q.k = m.conv_out + keys;
        q.v = m.conv_out + 2 * keys;
        q.stride = l.channels;
        q.rows = rows;
        q.heads = p.heads;
        q.dim_pad = p.dim_pad;
        q.vdim_pad = p.vdim_pad;
        q.state = p.state;
        q.chunk_states = m.chunk_states;
        q.control = s.control;
        q.capacity = p.capacity;
        q.out = b.linear_out;
        q.token.step = static_cast<const bf16*>(b.fused) + l.step_at;
        q.token.step_stride = l.in.out;
        q.token.bias = p.bias;
        q.token.rate = p.rate;
        q.token.skip = p.skip;
        q.token.key_heads = p.key_heads;
        q.token.ring_k = p.ring_k;
        q.token.ring_g = p.ring_g;
        q.token.ring_u = p.ring_u;
        q.token.totals = m.decay_totals;
        tick(s);
        int more = 0;
        launch_lightning_prompt(q, s.stream, pdl, &more);
        s.launches += size_t(more - 1);
      }
      StateFinishParams f = state_finish_params<bf16>(s, l, b);
      f.tail_rows = std::min(rows, p.taps - 1);
      f.tail = b.fused;
      f.tail_stride = l.in.out;
      f.channels = l.channels;
      f.raw_rows = l.raw_rows;
      f.raw = r.raw;
      f.control = s.control;
      f.capacity = p.capacity;
      tick(s);
      launch_state_finish<bf16>(f, s.stream, pdl);
      return;
    }
  }
}

void enqueue_layered_segment(ei_session& s, int rows, size_t context) {
  ei_model& model = *s.model;
  const LayeredModel& m = *model.layered;
  LayeredSession& L = *s.layered;
  auto& ws = model.prompt;
  const bool pdl = true;
  const Buffers b{rows,         ws.step_tokens, m.residual, m.linear_out,    ws.normed, ws.qkv,
                  ws.attention, ws.gate_up,     ws.act,     m.second_normed, m.second};
  EmbedParams token{};
  token.tokens = ws.tokens;
  token.control = s.control;
  token.step_tokens = ws.step_tokens;
  token.vocab = int(model.config.vocab_size);
  token.rows = rows;
  token.capacity = int(s.capacity);
  enqueue_embed<bf16>(s, b, token);

  const auto sums = [&](const PreparedLinear& w, const bf16* x, float* partial) {
    const int ksplit = prompt_gemm_ksplit(rows, w.out, w.in, model.multiprocessors, ws.partial_bytes);
    run_prompt_linear(s, w, x, rows, nullptr, pdl, ksplit, 0, partial);
    return ksplit;
  };
  for (size_t run = 0; run < m.runs.size(); ++run) {
    const LayeredModel::Layer& l = m.layers[m.runs[run].layer];
    enqueue_mixer_segment(s, l, L.runs[run], b, context);
    const bool feeds = l.spec.mlp != EI_MLP_NONE;
    const auto activate = [&] {
      if (l.spec.mlp == EI_MLP_RELU_SQUARED) {
        run_prompt_linear(s, l.up, m.parallel ? m.second_normed : ws.normed, rows, ws.act, pdl);
        return;
      }
      run_prompt_linear(s, l.gate_up, m.parallel ? m.second_normed : ws.normed, rows, ws.gate_up, pdl);
      tick(s);
      launch_clamped_glu<bf16>(ws.gate_up, rows, l.ff_pad, l.gate_up.glu_limit, ws.act, model.multiprocessors, s.stream, pdl);
    };
    if (m.parallel) {
      const int mixed_ksplit = sums(l.out, ws.attention, m.mixed_partial);
      int fed_ksplit = 0;
      if (feeds) {
        activate();
        fed_ksplit = sums(l.down, ws.act, ws.partial);
      }
      enqueue_parallel_join<bf16>(s, b, run, m.mixed_partial, mixed_ksplit, feeds ? ws.partial : nullptr, fed_ksplit);
      continue;
    }
    int ksplit = sums(l.out, ws.attention, ws.partial);
    SublayerJoinParams j = join_params(s, b, ws.partial, ksplit);
    j.after = l.norm1b;
    if (feeds)
      j.before = l.norm2;
    else
      end_of_run(s, b, run, j);
    tick(s);
    launch_sublayer_join<bf16>(j, s.stream, pdl);
    if (!feeds) continue;
    activate();
    ksplit = sums(l.down, ws.act, ws.partial);
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
