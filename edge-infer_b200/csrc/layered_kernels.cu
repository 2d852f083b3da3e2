// Elementwise and per-row kernels of decoders described layer by layer: embedding, sublayer joins, the preparation of
// a mixer's heads, the end of a mixer, the gated recurrence, the clamped gated unit, and FP32 linears.
#include "layered_device.cuh"

#include <algorithm>
#include <cmath>
#include <stdexcept>

namespace ei {
namespace {

__device__ __forceinline__ float4 dynamic_tanh(const DynamicTanh& n, int i, float4 x) {
  const float4 w = load_quad(n.weight + i), b = load_quad(n.bias + i);
  return make_float4(fmaf(tanhf(n.alpha * x.x), w.x, b.x), fmaf(tanhf(n.alpha * x.y), w.y, b.y),
                     fmaf(tanhf(n.alpha * x.z), w.z, b.z), fmaf(tanhf(n.alpha * x.w), w.w, b.w));
}

constexpr int kEmbedThreads = 256;
template <typename T>
__global__ void __launch_bounds__(kEmbedThreads) layered_embed_kernel(const LayeredEmbedParams p) {
  __shared__ uint32_t token_shared;
  grid_dependency_wait();
  const int row = blockIdx.x;
  if (threadIdx.x == 0) token_shared = take_step_token(p.token, row);
  __syncthreads();
  grid_launch_dependents();
  const uint32_t token = token_shared < uint32_t(p.token.vocab) ? token_shared : 0u;
  T* normed = static_cast<T*>(p.normed) + size_t(row) * p.normed_stride;
  for (int i = threadIdx.x * 4; i < p.normed_stride; i += kEmbedThreads * 4) {
    float4 out = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (i < p.residual_stride) {
      float4 x = load_quad(p.table + size_t(token) * p.residual_stride + i);
      if (p.vector) x = add(x, load_quad(p.vector + i));
      *reinterpret_cast<float4*>(p.residual + size_t(row) * p.residual_stride + i) = x;
      out = dynamic_tanh(p.norm, i, x);
    }
    store_quad(normed + i, out);
  }
}

// Four columns per thread, rows along y.
constexpr int kJoinThreads = 128;
template <typename T>
__global__ void __launch_bounds__(kJoinThreads) sublayer_join_kernel(const SublayerJoinParams p) {
  const int i = (blockIdx.x * kJoinThreads + threadIdx.x) * 4;
  const bool live = i < p.residual_stride;
  // Norm vectors do not come from the preceding kernel.
  float4 wa = make_float4(0.0f, 0.0f, 0.0f, 0.0f), ba = wa, wb = wa, bb = wa;
  if (live) {
    wa = load_quad(p.after.weight + i);
    ba = load_quad(p.after.bias + i);
    wb = load_quad(p.before.weight + i);
    bb = load_quad(p.before.bias + i);
  }
  grid_dependency_wait();
  grid_launch_dependents();
  if (i >= p.normed_stride) return;
  for (int row = blockIdx.y; row < p.rows; row += gridDim.y) {
    float4 out = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (live) {
      const size_t at = size_t(row) * p.residual_stride + i;
      const size_t slice = size_t(p.rows) * p.residual_stride;
      float4 y = *reinterpret_cast<const float4*>(p.partial + at);
      for (int s = 1; s < p.ksplit; ++s) y = add(y, *reinterpret_cast<const float4*>(p.partial + s * slice + at));
      float4 x = *reinterpret_cast<const float4*>(p.residual + at);
      x.x += fmaf(tanhf(p.after.alpha * y.x), wa.x, ba.x);
      x.y += fmaf(tanhf(p.after.alpha * y.y), wa.y, ba.y);
      x.z += fmaf(tanhf(p.after.alpha * y.z), wa.z, ba.z);
      x.w += fmaf(tanhf(p.after.alpha * y.w), wa.w, ba.w);
      if (p.tap) {
        float* tap = p.tap + size_t(row) * p.tap_width;
        const float values[4] = {x.x, x.y, x.z, x.w};
        for (int j = 0; j < 4; ++j)
          if (i + j < p.tap_width) tap[i + j] = values[j];
      }
      if (p.inject.table) {
        const uint32_t token = p.inject.tokens[row];
        x = add(x, load_quad(p.inject.table + size_t(token < uint32_t(p.inject.vocab) ? token : 0u) * p.residual_stride + i));
      }
      if (p.inject.vector) x = add(x, load_quad(p.inject.vector + i));
      *reinterpret_cast<float4*>(p.residual + at) = x;
      out = make_float4(fmaf(tanhf(p.before.alpha * x.x), wb.x, bb.x), fmaf(tanhf(p.before.alpha * x.y), wb.y, bb.y),
                        fmaf(tanhf(p.before.alpha * x.z), wb.z, bb.z), fmaf(tanhf(p.before.alpha * x.w), wb.w, bb.w));
    }
    store_quad(static_cast<T*>(p.normed) + size_t(row) * p.normed_stride + i, out);
  }
}

// One warp per (row, unit); units in the order of the fused projection: q heads, k heads, v heads, then the linear
// attention's q, k and v heads.
template <typename T>
__global__ void __launch_bounds__(128) mixer_prepare_kernel(const MixerPrepareParams p) {
  const int warp = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int units = p.heads + 2 * p.kv_heads + 3 * p.lin_heads;
  const int context = p.control->context;  // written by the previous step
  grid_dependency_wait();
  grid_launch_dependents();
  if (warp >= p.rows * units || context < 0 || context + p.rows > p.capacity) return;
  const int row = warp / units;
  int unit = warp - row * units;
  const int position = context + row;
  T* x = static_cast<T*>(p.fused) + size_t(row) * p.stride;

  if (unit < p.heads + p.kv_heads) {  // rotation of a q or k head; k goes to the cache
    const bool key = unit >= p.heads;
    x += size_t(unit) * p.dim_pad;
    T* to = key ? static_cast<T*>(p.k_cache) + (size_t(position) * p.kv_heads + (unit - p.heads)) * p.dim_pad : x;
    const int half = p.rot_dims >> 1;
    const float2* turn = p.rotation + size_t(position) * half;
    if (half % 4 == 0) {
      for (int i = lane * 4; i < half; i += 128) {
        const float4 u = load_quad(x + i), v = load_quad(x + i + half);
        const float4 t01 = *reinterpret_cast<const float4*>(turn + i), t23 = *reinterpret_cast<const float4*>(turn + i + 2);
        store_quad(to + i, make_float4(u.x * t01.x - v.x * t01.y, u.y * t01.z - v.y * t01.w, u.z * t23.x - v.z * t23.y,
                                       u.w * t23.z - v.w * t23.w));
        store_quad(to + i + half, make_float4(v.x * t01.x + u.x * t01.y, v.y * t01.z + u.y * t01.w, v.z * t23.x + u.z * t23.y,
                                              v.w * t23.z + u.w * t23.w));
      }
    } else if (half & 1) {
      for (int i = lane; i < half; i += 32) {
        const float u = value_of(x[i]), v = value_of(x[i + half]);
        const float2 t = turn[i];
        store_value(to + i, u * t.x - v * t.y);
        store_value(to + i + half, v * t.x + u * t.y);
      }
    } else {
      for (int i = lane * 2; i < half; i += 64) {
        const float2 u = load_pair(x + i), v = load_pair(x + i + half);
        const float2 t0 = turn[i], t1 = turn[i + 1];
        store_pair(to + i, u.x * t0.x - v.x * t0.y, u.y * t1.x - v.y * t1.y);
        store_pair(to + i + half, v.x * t0.x + u.x * t0.y, v.y * t1.x + u.y * t1.y);
      }
    }
    if (key)
      for (int i = p.rot_dims + lane * 2; i < p.dim_pad; i += 64) {
        const float2 v = load_pair(x + i);
        store_pair(to + i, v.x, v.y);
      }
    return;
  }
  unit -= p.heads + p.kv_heads;
  x += size_t(p.heads + p.kv_heads) * p.dim_pad;
  if (unit < p.kv_heads) {  // value norm, into the cache
    x += size_t(unit) * p.vdim_pad;
    T* to = static_cast<T*>(p.v_cache) + (size_t(position) * p.kv_heads + unit) * p.vdim_pad;
    float sum = 0.0f;
    for (int i = lane * 4; i < p.vdim_pad; i += 128) {
      const float4 v = load_quad(x + i);
      sum = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, sum))));
    }
    const float inverse = 1.0f / sqrtf(warp_sum(sum) / float(p.vdim) + p.eps);
    for (int i = lane * 4; i < p.vdim_pad; i += 128) {
      const float4 v = load_quad(x + i);
      store_quad(to + i, make_float4(v.x * inverse, v.y * inverse, v.z * inverse, v.w * inverse));
    }
    return;
  }
  unit -= p.kv_heads;
  x += size_t(p.kv_heads) * p.vdim_pad;
  const int kind = unit / p.lin_heads, head = unit - kind * p.lin_heads;  // 0 q, 1 k, 2 v
  const int pad = kind == 2 ? p.lin_vdim_pad : p.lin_dim_pad;
  x += size_t(min(kind, 2)) * p.lin_heads * p.lin_dim_pad + size_t(head) * pad;
  T* ring = nullptr;
  if (p.ring_k && kind > 0)
    ring = static_cast<T*>(kind == 1 ? p.ring_k : p.ring_v) + (size_t(position & (kRingRows - 1)) * p.lin_heads + head) * pad;
  for (int i = lane * 4; i < pad; i += 128) {
    float4 v = load_quad(x + i);
    v = make_float4(silu_for<T>(v.x), silu_for<T>(v.y), silu_for<T>(v.z), silu_for<T>(v.w));
    store_quad(x + i, v);
    if (ring) store_quad(ring + i, v);
  }
}

// Blocks [0, rows * heads) merge one (row, head) of the split attention (when asked to); the last `rows` blocks finish
// one row of the linear attention: RMS norm over all heads, weight, sigmoid gate, scale. At most 64 splits.
constexpr int kFinishWarps = 8;
constexpr int kFinishThreads = kFinishWarps * 32;
constexpr int kFinishHeld = 4;  // quads of a row a thread keeps between the two passes over it
template <typename T>
__global__ void __launch_bounds__(kFinishThreads) mixer_finish_kernel(const MixerFinishParams p) {
  __shared__ float weights[64];
  __shared__ float shared[2 * kFinishWarps];
  __shared__ float4 parts[kFinishWarps][32];
  const int merges = p.merge ? p.rows * p.attention.heads : 0;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  if (int(blockIdx.x) < merges) {
    const SizedAttentionParams& a = p.attention;
    const int offset = *a.device_offset;
    grid_dependency_wait();
    grid_launch_dependents();
    if (offset < 0 || offset + p.rows > a.capacity) return;
    const int slot = blockIdx.x, row = slot / a.heads, head = slot - row * a.heads;
    const int slots = p.rows * a.heads, pitch = a.vdim_pad + 4;
    const int splits = min(64, (offset + p.rows + a.chunk - 1) / a.chunk);
    const float* base = a.scratch + size_t(slot) * pitch;
    const size_t step = size_t(slots) * pitch;
    // A warp's splits are w, w + 8, ...; lane l owns columns 4 l .. 4 l + 3 of each 128. The first 128 columns are
    // requested together with the maxima and sums.
    float4 values[64 / kFinishWarps];
    auto request = [&](int column) {
#pragma unroll
      for (int i = 0; i < 64 / kFinishWarps; ++i) {
        const int s = warp + kFinishWarps * i;
        values[i] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (s < splits && column < a.vdim_pad) values[i] = *reinterpret_cast<const float4*>(base + s * step + column);
      }
    };
    request(lane * 4);
    float m = -INFINITY, l = 0.0f;
    if (int(threadIdx.x) < splits) {
      const float2 ml = *reinterpret_cast<const float2*>(base + threadIdx.x * step + a.vdim_pad);
      m = ml.x;
      l = ml.y;
    }
    const float sink = a.sink ? a.sink[head] : -INFINITY;
    if (warp < 2) {
      const float top = warp_max(m);
      if (lane == 0) shared[warp] = top;
    }
    __syncthreads();
    const float top = fmaxf(fmaxf(shared[0], shared[1]), sink);
    if (warp < 2) {
      const float weight = m == -INFINITY ? 0.0f : expf(m - top);
      weights[threadIdx.x] = weight;
      const float part = warp_sum(l * weight);
      if (lane == 0) shared[2 + warp] = part;
    }
    __syncthreads();
    const float denominator = shared[2] + shared[3] + (a.sink ? expf(sink - top) : 0.0f);
    const float factor = denominator > 0.0f ? a.out_scale / denominator : 0.0f;
    T* out = static_cast<T*>(a.out) + size_t(row) * a.out_stride + size_t(head) * a.vdim_pad;
    for (int first = 0; first < a.vdim_pad; first += 128) {
      const int column = first + lane * 4;
      if (first) request(column);
      float4 sum = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
      for (int i = 0; i < 64 / kFinishWarps; ++i) {
        const int s = warp + kFinishWarps * i;
        const float w = s < splits ? weights[s] : 0.0f;
        sum = make_float4(fmaf(values[i].x, w, sum.x), fmaf(values[i].y, w, sum.y), fmaf(values[i].z, w, sum.z),
                          fmaf(values[i].w, w, sum.w));
      }
      parts[warp][lane] = sum;
      __syncthreads();
      if (warp == 0 && column < a.vdim_pad) {
        for (int w = 1; w < kFinishWarps; ++w) sum = add(sum, parts[w][lane]);
        store_quad(out + column, make_float4(sum.x * factor, sum.y * factor, sum.z * factor, sum.w * factor));
      }
      __syncthreads();
    }
    return;
  }
  const int row = int(blockIdx.x) - merges;
  const int width = p.lin_heads * p.lin_vdim_pad;
  const T* gate = static_cast<const T*>(p.gate) + size_t(row) * p.gate_stride;
  const float* x = p.lin_out + size_t(row) * width;
  T* out = static_cast<T*>(p.out) + size_t(row) * p.out_stride + p.lin_offset;
  grid_dependency_wait();
  grid_launch_dependents();
  float4 held[kFinishHeld], gates[kFinishHeld];
  float sum = 0.0f;
#pragma unroll
  for (int j = 0; j < kFinishHeld; ++j) {
    const int i = (threadIdx.x + j * kFinishThreads) * 4;
    held[j] = gates[j] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (i < width) {
      held[j] = *reinterpret_cast<const float4*>(x + i);
      gates[j] = load_quad(gate + i);
    }
    sum = fmaf(held[j].x, held[j].x, fmaf(held[j].y, held[j].y, fmaf(held[j].z, held[j].z, fmaf(held[j].w, held[j].w, sum))));
  }
  for (int i = (threadIdx.x + kFinishHeld * kFinishThreads) * 4; i < width; i += kFinishThreads * 4) {
    const float4 v = *reinterpret_cast<const float4*>(x + i);
    sum = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, sum))));
  }
  const float mean = block_total(sum, shared) / (float(p.lin_heads) * float(p.lin_vdim));
  const float factor = p.lin_scale / sqrtf(mean + p.eps);
  const int end = p.out_stride - p.lin_offset;  // the columns behind the heads pad the projection's input
  auto finish = [&](int i, float4 v, float4 z) {
    float4 y = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (i < width) {
      const float4 w = load_quad(p.norm + i);
      y = make_float4(v.x * factor * w.x * sigmoid_for<T>(z.x), v.y * factor * w.y * sigmoid_for<T>(z.y),
                      v.z * factor * w.z * sigmoid_for<T>(z.z), v.w * factor * w.w * sigmoid_for<T>(z.w));
    }
    store_quad(out + i, y);
  };
#pragma unroll
  for (int j = 0; j < kFinishHeld; ++j) {
    const int i = (threadIdx.x + j * kFinishThreads) * 4;
    if (i < end) finish(i, held[j], gates[j]);
  }
  for (int i = (threadIdx.x + kFinishHeld * kFinishThreads) * 4; i < end; i += kFinishThreads * 4) {
    const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    finish(i, i < width ? *reinterpret_cast<const float4*>(x + i) : zero, i < width ? load_quad(gate + i) : zero);
  }
}

__device__ __forceinline__ float min_gru_candidate(float u) { return u >= 0.0f ? u + 0.5f : sigmoid_value(u); }

// One thread per channel. Pending rows are folded into the state; the step's own rows stay pending in the ring.
template <typename T>
__global__ void __launch_bounds__(128) min_gru_step_kernel(const MinGruParams p) {
  const int channel = blockIdx.x * 128 + threadIdx.x;
  const int context = p.control->context, base = p.control->state_base;
  const bool runs = context >= 0 && context + p.rows <= p.capacity;
  const int pending = min(kPendingRows, max(0, context - base));
  float s = 0.0f;
  if (runs && channel < p.width_pad) {  // the ring and the state were written by earlier steps
    if (base > 0) s = p.state[channel];
    for (int i = 0; i < pending; ++i) {
      const size_t at = size_t((base + i) & (kRingRows - 1)) * p.width_pad + channel;
      const float z = p.ring_gate[at];
      s = (1.0f - z) * s + z * p.ring_candidate[at];
    }
  }
  grid_dependency_wait();
  grid_launch_dependents();
  if (!runs || channel >= p.out_stride) return;
  T* out = static_cast<T*>(p.out) + channel;
  if (channel >= p.width_pad) {
    for (int r = 0; r < p.rows; ++r) store_value(out + size_t(r) * p.out_stride, 0.0f);
    return;
  }
  if (pending) p.state[channel] = s;
  for (int r = 0; r < p.rows; ++r) {
    const T* x = static_cast<const T*>(p.fused) + size_t(r) * p.stride + channel;
    const float z = sigmoid_value(value_of(x[0])), candidate = min_gru_candidate(value_of(x[p.width_pad]));
    const size_t at = size_t((context + r) & (kRingRows - 1)) * p.width_pad + channel;
    p.ring_gate[at] = z;
    p.ring_candidate[at] = candidate;
    s = (1.0f - z) * s + z * candidate;
    store_value(out + size_t(r) * p.out_stride, s * silu_exact(value_of(x[2 * p.width_pad])));
  }
}

// A prompt segment runs in stretches of 32 rows, two channels per thread. The first kernel reduces every stretch to
// (product of 1 - z, value from zero) and leaves the state with its pending rows folded in behind the stretches; the
// second chains the stretches before its own from that state and emits the rows, the last stretch writes the new state.
constexpr int kStretch = kMinGruStretch;
constexpr int kGruThreads = 64;
template <bool kEmit>
__global__ void __launch_bounds__(kGruThreads) min_gru_prompt_kernel(const MinGruParams p) {
  const int context = p.control->context, base = p.control->state_base;
  const bool runs = context >= 0 && context + p.rows <= p.capacity;
  grid_dependency_wait();
  grid_launch_dependents();
  const int channel = (blockIdx.x * kGruThreads + threadIdx.x) * 2;
  if (!runs || channel >= p.out_stride) return;
  const int stretch = blockIdx.y, begin = stretch * kStretch, end = min(p.rows, begin + kStretch);
  bf16* out = static_cast<bf16*>(p.out) + channel;
  if (channel >= p.width_pad) {
    if (kEmit)
      for (int t = begin; t < end; ++t) store_pair(out + size_t(t) * p.out_stride, 0.0f, 0.0f);
    return;
  }
  float s0 = 0.0f, s1 = 0.0f, a0 = 1.0f, a1 = 1.0f;
  float4* stretches = reinterpret_cast<float4*>(p.stretches) + channel / 2;
  float4* folded = stretches + size_t(gridDim.y) * (p.width_pad / 2);
  if (!kEmit && stretch == 0) {
    float2 s = base > 0 ? load_pair(p.state + channel) : make_float2(0.0f, 0.0f);
    const int pending = min(kPendingRows, max(0, context - base));
    for (int i = 0; i < pending; ++i) {
      const size_t at = size_t((base + i) & (kRingRows - 1)) * p.width_pad + channel;
      const float2 z = load_pair(p.ring_gate + at), c = load_pair(p.ring_candidate + at);
      s.x = (1.0f - z.x) * s.x + z.x * c.x;
      s.y = (1.0f - z.y) * s.y + z.y * c.y;
    }
    *folded = make_float4(s.x, s.y, 0.0f, 0.0f);
  }
  if (kEmit) {
    s0 = folded->x;
    s1 = folded->y;
#pragma unroll 8
    for (int i = 0; i < stretch; ++i) {
      const float4 r = stretches[size_t(i) * (p.width_pad / 2)];
      s0 = fmaf(r.x, s0, r.z);
      s1 = fmaf(r.y, s1, r.w);
    }
  }
  // Eight rows are requested at once: stores to `out` would otherwise keep the next row's loads behind them.
  constexpr int kBatch = 8;
  const uint32_t* x = reinterpret_cast<const uint32_t*>(static_cast<const bf16*>(p.fused) + size_t(begin) * p.stride + channel);
  const int pitch = p.stride / 2, section = p.width_pad / 2;
  for (int t = begin; t < end; t += kBatch, x += size_t(kBatch) * pitch) {
    uint32_t gates[kBatch], candidates[kBatch], outputs[kBatch];
#pragma unroll
    for (int j = 0; j < kBatch; ++j) {
      if (t + j < end) {
        gates[j] = __ldg(x + size_t(j) * pitch);
        candidates[j] = __ldg(x + size_t(j) * pitch + section);
        if (kEmit) outputs[j] = __ldg(x + size_t(j) * pitch + 2 * section);
      }
    }
#pragma unroll
    for (int j = 0; j < kBatch; ++j) {
      if (t + j < end) {
        const float z0 = quick_sigmoid(bf16_lo(gates[j])), z1 = quick_sigmoid(bf16_hi(gates[j]));
        s0 = (1.0f - z0) * s0 + z0 * quick_candidate(bf16_lo(candidates[j]));
        s1 = (1.0f - z1) * s1 + z1 * quick_candidate(bf16_hi(candidates[j]));
        if (kEmit) {
          const float g0 = bf16_lo(outputs[j]), g1 = bf16_hi(outputs[j]);
          store_pair(out + size_t(t + j) * p.out_stride, s0 * g0 * quick_sigmoid(g0), s1 * g1 * quick_sigmoid(g1));
        } else {
          a0 *= 1.0f - z0;
          a1 *= 1.0f - z1;
        }
      }
    }
  }
  if (!kEmit)
    stretches[size_t(stretch) * (p.width_pad / 2)] = make_float4(a0, a1, s0, s1);
  else if (end == p.rows)
    store_pair(p.state + channel, s0, s1);
}

template <typename T>
__global__ void __launch_bounds__(256) clamped_glu_kernel(const T* gate_up, int rows, int ff, float limit, T* out) {
  grid_dependency_wait();
  grid_launch_dependents();
  const int per_row = ff / 4;
  const long long total = (long long)rows * per_row;
  for (long long i = blockIdx.x * 256ll + threadIdx.x; i < total; i += gridDim.x * 256ll) {
    const int row = int(i / per_row), n = int(i - (long long)row * per_row) * 4;
    const float4 g = load_quad(gate_up + size_t(row) * 2 * ff + n), u = load_quad(gate_up + size_t(row) * 2 * ff + ff + n);
    store_quad(out + size_t(row) * ff + n,
               make_float4(clamped_glu_value(g.x, u.x, limit), clamped_glu_value(g.y, u.y, limit),
                           clamped_glu_value(g.z, u.z, limit), clamped_glu_value(g.w, u.w, limit)));
  }
}

template <typename T>
__global__ void __launch_bounds__(256) gather_rows_kernel(const T* source, const int32_t* index, int stride, T* out) {
  const T* from = source + size_t(index[blockIdx.x]) * stride;
  for (int i = threadIdx.x; i < stride; i += 256) out[size_t(blockIdx.x) * stride + i] = from[i];
}

__global__ void __launch_bounds__(256) sum_partials_kernel(const float* partial, int ksplit, size_t count, float cap, float* out) {
  grid_dependency_wait();
  for (size_t i = size_t(blockIdx.x) * 256 + threadIdx.x; i < count; i += size_t(gridDim.x) * 256) {
    float sum = partial[i];
    for (int s = 1; s < ksplit; ++s) sum += partial[s * count + i];
    out[i] = cap > 0.0f ? cap * tanhf(sum / cap) : sum;
  }
}

// A warp per output feature, the rows' products summed lane by lane and then across the warp.
constexpr int kTrue32Tile = 256;
__global__ void __launch_bounds__(256) true32_linear_kernel(const float* x, int x_stride, int rows, const bf16* w,
                                                            const bf16* bias, int activation, int in, int out_features,
                                                            float* out) {
  __shared__ float tile[kMaxRows][kTrue32Tile];
  grid_dependency_wait();
  grid_launch_dependents();
  const int n = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  float acc[kMaxRows];
#pragma unroll
  for (int r = 0; r < kMaxRows; ++r) acc[r] = 0.0f;
  for (int first = 0; first < in; first += kTrue32Tile) {
    const int width = min(kTrue32Tile, in - first);
    __syncthreads();
    for (int i = threadIdx.x; i < rows * kTrue32Tile; i += 256) {
      const int r = i / kTrue32Tile, k = i - r * kTrue32Tile;
      tile[r][k] = k < width ? x[size_t(r) * x_stride + first + k] : 0.0f;
    }
    __syncthreads();
    if (n < out_features) {
      for (int k = lane; k < width; k += 32) {
        const float weight = __bfloat162float(w[size_t(n) * in + first + k]);
#pragma unroll
        for (int r = 0; r < kMaxRows; ++r)
          if (r < rows) acc[r] = fmaf(tile[r][k], weight, acc[r]);
      }
    }
  }
  if (n >= out_features) return;
#pragma unroll
  for (int r = 0; r < kMaxRows; ++r) {
    if (r < rows) {
      const float sum = warp_sum(acc[r]);
      if (lane == 0)
        out[size_t(r) * out_features + n] = activated_value(activation, sum + (bias ? __bfloat162float(bias[n]) : 0.0f));
    }
  }
}

__global__ void rotation_table_kernel(float2* table, size_t positions, const double* frequencies, int half, double length) {
  for (size_t i = size_t(blockIdx.x) * blockDim.x + threadIdx.x; i < positions * half; i += size_t(gridDim.x) * blockDim.x) {
    double s, c;
    sincos(double(i / half) * frequencies[i % half], &s, &c);
    table[i] = make_float2(float(c * length), float(s * length));
  }
}

}  // namespace

template <typename T>
void launch_layered_embed(const LayeredEmbedParams& p, cudaStream_t stream, bool pdl) {
  launch(layered_embed_kernel<T>, dim3(p.token.rows), dim3(kEmbedThreads), 0, stream, pdl, p);
}
template <typename T>
void launch_sublayer_join(const SublayerJoinParams& p, cudaStream_t stream, bool pdl) {
  const unsigned columns = unsigned((p.normed_stride / 4 + kJoinThreads - 1) / kJoinThreads);
  launch(sublayer_join_kernel<T>, dim3(columns, unsigned(std::min(p.rows, 1024))), dim3(kJoinThreads), 0, stream, pdl, p);
}
template <typename T>
void launch_mixer_prepare(const MixerPrepareParams& p, cudaStream_t stream, bool pdl) {
  const int warps = p.rows * (p.heads + 2 * p.kv_heads + 3 * p.lin_heads);
  launch(mixer_prepare_kernel<T>, dim3(unsigned((warps + 3) / 4)), dim3(128), 0, stream, pdl, p);
}
template <typename T>
void launch_mixer_finish(const MixerFinishParams& p, cudaStream_t stream, bool pdl) {
  const int blocks = p.rows + (p.merge ? p.rows * p.attention.heads : 0);
  launch(mixer_finish_kernel<T>, dim3(unsigned(blocks)), dim3(kFinishThreads), 0, stream, pdl, p);
}
template <typename T>
void launch_min_gru_step(const MinGruParams& p, cudaStream_t stream, bool pdl) {
  launch(min_gru_step_kernel<T>, dim3(unsigned((p.out_stride + 127) / 128)), dim3(128), 0, stream, pdl, p);
}
void launch_min_gru_prompt(const MinGruParams& p, cudaStream_t stream, bool pdl) {
  const dim3 grid(unsigned((p.out_stride / 2 + kGruThreads - 1) / kGruThreads), unsigned((p.rows + kStretch - 1) / kStretch));
  launch(min_gru_prompt_kernel<false>, grid, dim3(kGruThreads), 0, stream, pdl, p);
  launch(min_gru_prompt_kernel<true>, grid, dim3(kGruThreads), 0, stream, pdl, p);
}
template <typename T>
void launch_clamped_glu(const T* gate_up, int rows, int ff, float limit, T* out, int multiprocessors,
                        cudaStream_t stream, bool pdl) {
  const long long quads = (long long)rows * ff / 4;
  const unsigned blocks = unsigned(std::max(1ll, std::min((quads + 255) / 256, (long long)multiprocessors * 8)));
  launch(clamped_glu_kernel<T>, dim3(blocks), dim3(256), 0, stream, pdl, gate_up, rows, ff, limit, out);
}
template <typename T>
void launch_gather_rows(const T* source, const int32_t* index, int count, int stride, T* out, cudaStream_t stream) {
  launch(gather_rows_kernel<T>, dim3(count), dim3(256), 0, stream, false, source, index, stride, out);
}
void launch_sum_partials(const float* partial, int ksplit, size_t count, float cap, float* out, int multiprocessors,
                         cudaStream_t stream, bool pdl) {
  const unsigned blocks = unsigned(std::max<size_t>(1, std::min((count + 255) / 256, size_t(multiprocessors) * 8)));
  launch(sum_partials_kernel, dim3(blocks), dim3(256), 0, stream, pdl, partial, ksplit, count, cap, out);
}
void launch_true32_linear(const float* x, int x_stride, int rows, const PreparedLinear& w, float* out, cudaStream_t stream,
                          bool pdl) {
  if (rows < 1 || rows > kMaxRows) throw std::invalid_argument("32-bit linear takes 1..16 rows");
  launch(true32_linear_kernel, dim3(unsigned((w.out + 7) / 8)), dim3(256), 0, stream, pdl, x, x_stride, rows, w.dense, w.bias,
         w.activation, w.in, w.out, out);
}
void launch_rotation_table(float2* table, size_t positions, const double* frequencies, int half, double length,
                           cudaStream_t stream) {
  const size_t count = positions * half;
  if (!count) return;
  rotation_table_kernel<<<unsigned(std::min<size_t>((count + 255) / 256, 4096)), 256, 0, stream>>>(table, positions, frequencies,
                                                                                                   half, length);
  check_launch();
}

template void launch_layered_embed<bf16>(const LayeredEmbedParams&, cudaStream_t, bool);
template void launch_layered_embed<float>(const LayeredEmbedParams&, cudaStream_t, bool);
template void launch_sublayer_join<bf16>(const SublayerJoinParams&, cudaStream_t, bool);
template void launch_sublayer_join<float>(const SublayerJoinParams&, cudaStream_t, bool);
template void launch_mixer_prepare<bf16>(const MixerPrepareParams&, cudaStream_t, bool);
template void launch_mixer_prepare<float>(const MixerPrepareParams&, cudaStream_t, bool);
template void launch_mixer_finish<bf16>(const MixerFinishParams&, cudaStream_t, bool);
template void launch_mixer_finish<float>(const MixerFinishParams&, cudaStream_t, bool);
template void launch_min_gru_step<bf16>(const MinGruParams&, cudaStream_t, bool);
template void launch_min_gru_step<float>(const MinGruParams&, cudaStream_t, bool);
template void launch_clamped_glu<bf16>(const bf16*, int, int, float, bf16*, int, cudaStream_t, bool);
template void launch_clamped_glu<float>(const float*, int, int, float, float*, int, cudaStream_t, bool);
template void launch_gather_rows<bf16>(const bf16*, const int32_t*, int, int, bf16*, cudaStream_t);
template void launch_gather_rows<float>(const float*, const int32_t*, int, int, float*, cudaStream_t);

}  // namespace ei
