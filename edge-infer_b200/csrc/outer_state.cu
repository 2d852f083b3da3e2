// Recurrences over one FP32 matrix per head, S (key size x value size): S <- g S, S <- S + k u^T, out = S^T q.
//
// Two rules for the written vector u: the gated delta rule u = beta (v - S^T k) with one decay per key channel, and a
// state-space layer's u = t v with one decay per head. q, k and v come out of a short causal convolution and SiLU.
//
// A step of at most 16 rows leaves its rows pending, as linear attention does (lightning.cu): the ring keeps every row's
// k, g and u, so the next step rebuilds the state from those rows that were kept by plain rank-one updates, without
// running the delta rule again. The convolution's inputs sit in a ring of their own, by position.
#include "layered_device.cuh"

#include <algorithm>
#include <stdexcept>

namespace ei {
namespace {

// One warp per (row, unit): q heads, k heads, v heads (convolution, SiLU, unit length), then the decays - per head for the
// delta rule, 32 heads at a time otherwise. What does not come from the preceding kernel - weights, and the inputs of
// earlier steps - is requested before waiting for it. kTaps 0: any number of taps.
constexpr int kStrips = 4;  // strips of 32 channels in flight
template <typename T, int kTaps>
__global__ void __launch_bounds__(128) outer_prepare_kernel(const OuterStateParams p) {
  constexpr int kHeldTaps = kTaps ? kTaps : 1;
  const int warp = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int units = 2 * p.key_heads + p.heads + (p.delta ? p.heads : (p.heads + 31) / 32);
  const int context = p.control->context;  // written by the previous step
  const bool runs = warp < p.rows * units && context >= 0 && context + p.rows <= p.capacity;
  const int row = warp / units, position = context + row;
  int unit = warp - row * units;
  const int slot = position & (kRingRows - 1);
  const T* fused = static_cast<const T*>(p.fused);

  if (unit < 2 * p.key_heads + p.heads) {
    const int kind = unit < p.key_heads ? 0 : unit < 2 * p.key_heads ? 1 : 2;  // q, k, v
    const int head = unit - kind * p.key_heads, pad = kind == 2 ? p.vdim_pad : p.dim_pad;
    const int first = kind * p.key_heads * p.dim_pad + head * pad;
    const int channels = 2 * p.key_heads * p.dim_pad + p.heads * p.vdim_pad;
    T* raw = static_cast<T*>(p.raw);
    float weights[kStrips][kHeldTaps], inputs[kStrips][kHeldTaps], bias[kStrips];
    auto settled = [&](int chunk) {  // weights, and inputs of earlier steps
#pragma unroll
      for (int j = 0; j < kStrips; ++j) {
        const int c = chunk + lane + 32 * j;
        bias[j] = c < pad && p.conv_bias ? p.conv_bias[first + c] : 0.0f;
#pragma unroll
        for (int tap = 0; tap < kTaps; ++tap) {
          const int r = row - (kTaps - 1) + tap;
          weights[j][tap] = c < pad ? p.conv[size_t(tap) * channels + first + c] : 0.0f;
          inputs[j][tap] = 0.0f;
          if (runs && c < pad && r < 0 && context + r >= 0) inputs[j][tap] = value_of(raw[size_t((context + r) & (p.raw_rows - 1)) * channels + first + c]);
        }
      }
    };
    settled(0);
    grid_dependency_wait();
    grid_launch_dependents();
    if (!runs) return;
    float* to = kind == 0 ? p.q + size_t(row) * p.key_heads * p.dim_pad + head * pad
                : kind == 1 ? p.ring_k + size_t(slot) * p.key_heads * p.dim_pad + head * pad
                            : p.v + size_t(row) * p.heads * p.vdim_pad + head * pad;
    float values[kStrips], squares = 0.0f;
    auto convolve = [&](int chunk) {
#pragma unroll
      for (int j = 0; j < kStrips; ++j) {
        const int c = chunk + lane + 32 * j;
        float sum = bias[j];
        if (c < pad) {
          const int channel = first + c;
          const T own = fused[size_t(row) * p.stride + channel];
          if (kTaps) {
#pragma unroll
            for (int tap = 0; tap < kTaps; ++tap) {
              const int r = row - (kTaps - 1) + tap;
              const float x = tap == kTaps - 1 ? value_of(own) : r >= 0 ? value_of(fused[size_t(r) * p.stride + channel]) : inputs[j][tap];
              sum = fmaf(x, weights[j][tap], sum);
            }
          } else {
            for (int tap = 0; tap < p.taps; ++tap) {
              const int r = row - (p.taps - 1) + tap, at = context + r;
              if (at < 0) continue;
              const T x = r >= 0 ? fused[size_t(r) * p.stride + channel] : raw[size_t(at & (p.raw_rows - 1)) * channels + channel];
              sum = fmaf(value_of(x), p.conv[size_t(tap) * channels + channel], sum);
            }
          }
          raw[size_t(position & (p.raw_rows - 1)) * channels + channel] = own;
        }
        values[j] = c < pad ? silu_for<T>(sum) : 0.0f;
        squares = fmaf(values[j], values[j], squares);
      }
    };
    // Heads wider than the strips in flight: the rest is stored as it is and scaled once the length is known.
#pragma unroll 1
    for (int chunk = 32 * kStrips; chunk < pad; chunk += 32 * kStrips) {
      settled(chunk);
      convolve(chunk);
#pragma unroll
      for (int j = 0; j < kStrips; ++j)
        if (chunk + lane + 32 * j < pad) to[chunk + lane + 32 * j] = values[j];
    }
    if (pad > 32 * kStrips) settled(0);
    convolve(0);
    float scale = 1.0f;
    if (p.delta && kind < 2) {
      scale = 1.0f / sqrtf(warp_sum(squares) + 1e-6f);
      if (kind == 0) scale /= sqrtf(float(p.dim));
      for (int c = 32 * kStrips + lane; c < pad; c += 32) to[c] *= scale;  // written by this lane
    }
#pragma unroll
    for (int j = 0; j < kStrips; ++j)
      if (lane + 32 * j < pad) to[lane + 32 * j] = values[j] * scale;
    return;
  }
  unit -= 2 * p.key_heads + p.heads;
  const int head = p.delta ? unit : unit * 32 + lane;
  const float rate = head < p.heads ? p.rate[head] : 0.0f;
  const float bias = !p.delta && head < p.heads ? p.bias[head] : 0.0f;
  float biases[kStrips];  // delta rule: of this lane's first key channels
#pragma unroll
  for (int j = 0; j < kStrips; ++j)
    biases[j] = p.delta && head < p.heads && lane + 32 * j < p.dim_pad ? p.bias[head * p.dim_pad + lane + 32 * j] : 0.0f;
  grid_dependency_wait();
  grid_launch_dependents();
  if (!runs) return;
  const T* step = fused + size_t(row) * p.stride + p.step_at;
  if (p.delta) {
    const T* decay = static_cast<const T*>(p.decay) + size_t(row) * p.decay_stride + head * p.dim_pad;
    float* to = p.ring_g + (size_t(slot) * p.heads + head) * p.dim_pad;
    if (lane == 0) p.beta[size_t(row) * p.heads + head] = sigmoid_value(value_of(step[head]));
    auto decay_of = [&](int d, float b) { to[d] = expf(-rate * softplus_value(value_of(decay[d]) + b)); };
#pragma unroll
    for (int j = 0; j < kStrips; ++j)
      if (lane + 32 * j < p.dim_pad) decay_of(lane + 32 * j, biases[j]);
    for (int d = lane + 32 * kStrips; d < p.dim_pad; d += 32) decay_of(d, p.bias[head * p.dim_pad + d]);
    return;
  }
  if (head >= p.heads) return;
  const float t = softplus_value(value_of(step[head]) + bias);
  p.ring_g[size_t(slot) * p.heads + head] = expf(-rate * t);
  p.beta[size_t(row) * p.heads + head] = t;
}

// Block (head, slice of 16 values): a warp owns four values over all key channels, lane l the channels l, l + 32, ...
template <bool kDelta, int kParts>
__global__ void __launch_bounds__(128) outer_step_kernel(const OuterStateParams p) {
  const int head = blockIdx.x, slice = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int key_head = head / (p.heads / p.key_heads);
  const int key_width = p.key_heads * p.dim_pad, value_width = p.heads * p.vdim_pad;
  const int value = head * p.vdim_pad + slice * 16 + warp * 4;
  // Written by the previous step, several kernels ago: read, and the pending rows folded, before waiting.
  const int context = p.control->context, base = p.control->state_base;
  const bool runs = context >= 0 && context + p.rows <= p.capacity;
  const int pending = min(kPendingRows, max(0, context - base));
  float* state = p.state + ((size_t(head) * (p.vdim_pad / 16) + slice) * p.dim_pad) * 16 + warp * 4;
  float4 s[kParts];
#pragma unroll
  for (int i = 0; i < kParts; ++i) {
    const int d = lane + 32 * i;
    s[i] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (runs && base > 0 && d < p.dim_pad) s[i] = *reinterpret_cast<const float4*>(state + size_t(d) * 16);
  }
  const float* keys = p.ring_k + key_head * p.dim_pad;
  const float* decays = p.ring_g + (kDelta ? head * p.dim_pad : head);
  const int decay_width = kDelta ? p.heads * p.dim_pad : p.heads;
  if (runs && pending) {
    for (int j = 0; j < pending; ++j) {
      const int slot = (base + j) & (kRingRows - 1);
      const float4 u = *reinterpret_cast<const float4*>(p.ring_u + size_t(slot) * value_width + value);
      const float whole = kDelta ? 0.0f : decays[size_t(slot) * decay_width];
#pragma unroll
      for (int i = 0; i < kParts; ++i) {
        const int d = lane + 32 * i;
        if (d >= p.dim_pad) continue;
        const float k = keys[size_t(slot) * key_width + d], g = kDelta ? decays[size_t(slot) * decay_width + d] : whole;
        s[i] = make_float4(fmaf(k, u.x, g * s[i].x), fmaf(k, u.y, g * s[i].y), fmaf(k, u.z, g * s[i].z), fmaf(k, u.w, g * s[i].w));
      }
    }
#pragma unroll
    for (int i = 0; i < kParts; ++i)
      if (lane + 32 * i < p.dim_pad) *reinterpret_cast<float4*>(state + size_t(lane + 32 * i) * 16) = s[i];
  }
  grid_dependency_wait();
  grid_launch_dependents();
  if (!runs) return;
  for (int row = 0; row < p.rows; ++row) {
    const int slot = (context + row) & (kRingRows - 1);
    const float4 v = *reinterpret_cast<const float4*>(p.v + size_t(row) * value_width + value);
    const float rate = p.beta[size_t(row) * p.heads + head];
    const float whole = kDelta ? 0.0f : decays[size_t(slot) * decay_width];
    float k[kParts];
    float4 seen = make_float4(0.0f, 0.0f, 0.0f, 0.0f), read = seen;  // S^T k and S^T q after the decay
    float match = 0.0f;                                              // q . k
#pragma unroll
    for (int i = 0; i < kParts; ++i) {
      const int d = lane + 32 * i;
      k[i] = 0.0f;
      if (d >= p.dim_pad) continue;
      k[i] = keys[size_t(slot) * key_width + d];
      const float q = p.q[size_t(row) * key_width + key_head * p.dim_pad + d];
      const float g = kDelta ? decays[size_t(slot) * decay_width + d] : whole;
      s[i] = make_float4(g * s[i].x, g * s[i].y, g * s[i].z, g * s[i].w);
      if (kDelta) seen = make_float4(fmaf(k[i], s[i].x, seen.x), fmaf(k[i], s[i].y, seen.y), fmaf(k[i], s[i].z, seen.z), fmaf(k[i], s[i].w, seen.w));
      read = make_float4(fmaf(q, s[i].x, read.x), fmaf(q, s[i].y, read.y), fmaf(q, s[i].z, read.z), fmaf(q, s[i].w, read.w));
      match = fmaf(q, k[i], match);
    }
    if (kDelta) {
      seen.x = warp_sum(seen.x); seen.y = warp_sum(seen.y); seen.z = warp_sum(seen.z); seen.w = warp_sum(seen.w);
    }
    read.x = warp_sum(read.x); read.y = warp_sum(read.y); read.z = warp_sum(read.z); read.w = warp_sum(read.w);
    match = warp_sum(match);
    const float4 u = make_float4(rate * (v.x - seen.x), rate * (v.y - seen.y), rate * (v.z - seen.z), rate * (v.w - seen.w));
#pragma unroll
    for (int i = 0; i < kParts; ++i)
      s[i] = make_float4(fmaf(k[i], u.x, s[i].x), fmaf(k[i], u.y, s[i].y), fmaf(k[i], u.z, s[i].z), fmaf(k[i], u.w, s[i].w));
    if (lane == 0) {
      const float skip = p.skip ? p.skip[head] : 0.0f;
      *reinterpret_cast<float4*>(p.ring_u + size_t(slot) * value_width + value) = u;
      *reinterpret_cast<float4*>(p.out + size_t(row) * value_width + value) =
          make_float4(fmaf(match, u.x, fmaf(skip, v.x, read.x)), fmaf(match, u.y, fmaf(skip, v.y, read.y)),
                      fmaf(match, u.z, fmaf(skip, v.z, read.z)), fmaf(match, u.w, fmaf(skip, v.w, read.w)));
    }
  }
}

// A prompt segment's convolution: a warp takes eight rows of one head of q, k or v, kVector channels per lane at a time.
// kTaps 0: any number of taps.
constexpr int kConvRows = 8;
template <int kVector>
struct Packed {
  uint32_t pair[kVector / 2];
};
__device__ __forceinline__ Packed<4> packed_at(const bf16* p, Packed<4>) {
  const uint2 x = *reinterpret_cast<const uint2*>(p);
  return {{x.x, x.y}};
}
__device__ __forceinline__ Packed<2> packed_at(const bf16* p, Packed<2>) { return {{*reinterpret_cast<const uint32_t*>(p)}}; }
__device__ __forceinline__ void put_packed(bf16* p, Packed<4> x) { *reinterpret_cast<uint2*>(p) = make_uint2(x.pair[0], x.pair[1]); }
__device__ __forceinline__ void put_packed(bf16* p, Packed<2> x) { *reinterpret_cast<uint32_t*>(p) = x.pair[0]; }

template <int kTaps, int kVector>
__device__ __forceinline__ void conv_head(const OuterStateParams& p, bf16* out, float* inverse, int context, int begin, int unit, int lane) {
  using Vector = Packed<kVector>;
  const int kind = unit < p.key_heads ? 0 : unit < 2 * p.key_heads ? 1 : 2;  // q, k, v
  const int head = unit - kind * p.key_heads, pad = kind == 2 ? p.vdim_pad : p.dim_pad;
  const int first = kind * p.key_heads * p.dim_pad + head * pad;
  const int channels = 2 * p.key_heads * p.dim_pad + p.heads * p.vdim_pad;
  const bf16* fused = static_cast<const bf16*>(p.fused);
  const bf16* raw = static_cast<const bf16*>(p.raw);
  const int taps = kTaps ? kTaps : p.taps;
  float squares[kConvRows];
#pragma unroll
  for (int r = 0; r < kConvRows; ++r) squares[r] = 0.0f;
  for (int c = lane * kVector; c < pad; c += 32 * kVector) {
    const int channel = first + c;
    auto input = [&](int r) {
      if (r >= p.rows) return Vector{};
      if (r >= 0) return packed_at(fused + size_t(r) * p.stride + channel, Vector{});
      return context + r >= 0 ? packed_at(raw + size_t((context + r) & (p.raw_rows - 1)) * channels + channel, Vector{}) : Vector{};
    };
    auto weight = [&](int tap, float (&w)[kVector]) {
#pragma unroll
      for (int j = 0; j < kVector; j += 2) {
        const float2 x = load_pair(p.conv + size_t(tap) * channels + channel + j);
        w[j] = x.x;
        w[j + 1] = x.y;
      }
    };
    auto accumulate = [](float (&sum)[kVector], const Vector& x, const float (&w)[kVector]) {
#pragma unroll
      for (int j = 0; j < kVector; j += 2) {
        sum[j] = fmaf(bf16_lo(x.pair[j / 2]), w[j], sum[j]);
        sum[j + 1] = fmaf(bf16_hi(x.pair[j / 2]), w[j + 1], sum[j + 1]);
      }
    };
    auto finish = [&](int r, float (&sum)[kVector]) {
      if (begin + r >= p.rows) return;
      Vector y;
#pragma unroll
      for (int j = 0; j < kVector; j += 2) {
        const float a = sum[j], b = sum[j + 1];
        y.pair[j / 2] = pack_bf16(a * quick_sigmoid(a), b * quick_sigmoid(b));
        squares[r] = fmaf(bf16_lo(y.pair[j / 2]), bf16_lo(y.pair[j / 2]), fmaf(bf16_hi(y.pair[j / 2]), bf16_hi(y.pair[j / 2]), squares[r]));
      }
      put_packed(out + size_t(begin + r) * channels + channel, y);
    };
    float bias[kVector];
#pragma unroll
    for (int j = 0; j < kVector; ++j) bias[j] = p.conv_bias ? p.conv_bias[channel + j] : 0.0f;
    if (kTaps) {
      constexpr int kHeld = kTaps ? kTaps : 1;
      Vector window[kConvRows + kHeld - 1];
      float w[kHeld][kVector];
#pragma unroll
      for (int i = 0; i < kConvRows + kHeld - 1; ++i) window[i] = input(begin + i - (kHeld - 1));
#pragma unroll
      for (int tap = 0; tap < kHeld; ++tap) weight(tap, w[tap]);
#pragma unroll
      for (int r = 0; r < kConvRows; ++r) {
        float sum[kVector];
#pragma unroll
        for (int j = 0; j < kVector; ++j) sum[j] = bias[j];
#pragma unroll
        for (int tap = 0; tap < kHeld; ++tap) accumulate(sum, window[r + tap], w[tap]);
        finish(r, sum);
      }
    } else {
#pragma unroll
      for (int r = 0; r < kConvRows; ++r) {
        float sum[kVector], w[kVector];
#pragma unroll
        for (int j = 0; j < kVector; ++j) sum[j] = bias[j];
        for (int tap = 0; tap < taps; ++tap) {
          weight(tap, w);
          accumulate(sum, input(begin + r - (taps - 1) + tap), w);
        }
        finish(r, sum);
      }
    }
  }
  if (!p.delta || kind == 2) return;
#pragma unroll
  for (int r = 0; r < kConvRows; ++r) {
    float scale = 1.0f / sqrtf(warp_sum(squares[r]) + 1e-6f);
    if (kind == 0) scale /= sqrtf(float(p.dim));
    if (lane == 0 && begin + r < p.rows) inverse[size_t(begin + r) * 2 * p.key_heads + unit] = scale;
  }
}

template <int kTaps>
__global__ void __launch_bounds__(128, 5) outer_conv_kernel(const OuterStateParams p, bf16* out, float* inverse) {
  const int context = p.control->context;  // written by the previous step
  grid_dependency_wait();
  grid_launch_dependents();
  if (context < 0 || context + p.rows > p.capacity) return;
  const int units = 2 * p.key_heads + p.heads;
  const int warp = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int unit = warp % units, begin = warp / units * kConvRows;
  if (begin >= p.rows) return;
  if ((unit < 2 * p.key_heads ? p.dim_pad : p.vdim_pad) > 64)
    conv_head<kTaps, 4>(p, out, inverse, context, begin, unit, lane);
  else
    conv_head<kTaps, 2>(p, out, inverse, context, begin, unit, lane);
}

// One warp (kWide: one block) per (row, norm group). Values of a group are those of its heads side by side, without the
// heads' padding.
constexpr int kFinishHeld = 8;   // values a thread keeps between the two passes over a group
constexpr int kFinishQuads = 4;  // the same, four at a time
constexpr int kTailPiece = 128;
template <typename T, bool kWide>
__global__ void __launch_bounds__(256) state_finish_kernel(const StateFinishParams p) {
  __shared__ float shared[8];
  grid_dependency_wait();
  grid_launch_dependents();
  const int lanes = kWide ? blockDim.x : 32, lane = kWide ? threadIdx.x : threadIdx.x & 31;
  const int item = kWide ? blockIdx.x : blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (item >= p.rows * p.groups) {
    // Behind them: convolution inputs into the ring, kTailPiece channels per item.
    const int pieces = (p.channels + kTailPiece - 1) / kTailPiece, tail = item - p.rows * p.groups;
    const int back = tail / pieces, r = p.rows - 1 - back, context = p.control ? p.control->context : -1;
    if (back >= p.tail_rows || context < 0 || context + p.rows > p.capacity) return;
    const T* from = static_cast<const T*>(p.tail) + size_t(r) * p.tail_stride;
    T* to = static_cast<T*>(p.raw) + size_t((context + r) & (p.raw_rows - 1)) * p.channels;
    const int begin = (tail - back * pieces) * kTailPiece, end = min(p.channels, begin + kTailPiece);
    for (int i = begin + lane * 2; i < end; i += lanes * 2) {
      const float2 v = load_pair(from + i);
      store_pair(to + i, v.x, v.y);
    }
    return;
  }
  const int row = item / p.groups, group = item - row * p.groups;
  const int length = p.heads * p.vdim / p.groups, first = group * length;
  const int width = p.heads * p.vdim_pad;
  const bool packed = p.vdim == p.vdim_pad;
  const float* in = p.in + size_t(row) * width;
  const T* gate = static_cast<const T*>(p.gate) + size_t(row) * p.gate_stride;
  T* out = static_cast<T*>(p.out) + size_t(row) * p.out_stride;
  auto column = [&](int e) { return packed ? first + e : (first + e) / p.vdim * p.vdim_pad + (first + e) % p.vdim; };
  if (packed && length % 4 == 0) {  // four values at a time
    auto gated = [&](float4 x, float4 z) {
      return p.gate_first ? make_float4(x.x * silu_for<T>(z.x), x.y * silu_for<T>(z.y), x.z * silu_for<T>(z.z), x.w * silu_for<T>(z.w)) : x;
    };
    float4 x[kFinishQuads], z[kFinishQuads];
    float squares = 0.0f;
#pragma unroll
    for (int j = 0; j < kFinishQuads; ++j) {
      const int e = (lane + j * lanes) * 4;
      x[j] = z[j] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
      if (e < length) {
        x[j] = *reinterpret_cast<const float4*>(in + first + e);
        z[j] = load_quad(gate + first + e);
      }
    }
#pragma unroll
    for (int j = 0; j < kFinishQuads; ++j) {
      x[j] = gated(x[j], z[j]);
      squares = fmaf(x[j].x, x[j].x, fmaf(x[j].y, x[j].y, fmaf(x[j].z, x[j].z, fmaf(x[j].w, x[j].w, squares))));
    }
    for (int e = (lane + kFinishQuads * lanes) * 4; e < length; e += lanes * 4) {
      const float4 y = gated(*reinterpret_cast<const float4*>(in + first + e), load_quad(gate + first + e));
      squares = fmaf(y.x, y.x, fmaf(y.y, y.y, fmaf(y.z, y.z, fmaf(y.w, y.w, squares))));
    }
    const float scale = 1.0f / sqrtf((kWide ? block_total(squares, shared) : warp_sum(squares)) / float(length) + p.eps);
    auto finish = [&](int e, float4 y, float4 gates) {
      const float4 w = load_quad(p.norm + first + e);
      y = make_float4(y.x * scale * w.x, y.y * scale * w.y, y.z * scale * w.z, y.w * scale * w.w);
      if (!p.gate_first)
        y = make_float4(y.x * sigmoid_for<T>(gates.x), y.y * sigmoid_for<T>(gates.y), y.z * sigmoid_for<T>(gates.z), y.w * sigmoid_for<T>(gates.w));
      store_quad(out + first + e, y);
    };
#pragma unroll
    for (int j = 0; j < kFinishQuads; ++j) {
      const int e = (lane + j * lanes) * 4;
      if (e < length) finish(e, x[j], z[j]);
    }
    for (int e = (lane + kFinishQuads * lanes) * 4; e < length; e += lanes * 4) {
      const float4 gates = load_quad(gate + first + e);
      finish(e, gated(*reinterpret_cast<const float4*>(in + first + e), gates), gates);
    }
    if (group == 0)
      for (int at = width + lane; at < p.out_stride; at += lanes) store_value(out + at, 0.0f);
    return;
  }
  auto value = [&](int at, float z) { return p.gate_first ? in[at] * silu_for<T>(z) : in[at]; };
  float held[kFinishHeld], gates[kFinishHeld], sum = 0.0f;
#pragma unroll
  for (int j = 0; j < kFinishHeld; ++j) {
    const int e = lane + j * lanes;
    held[j] = gates[j] = 0.0f;
    if (e < length) {
      const int at = column(e);
      gates[j] = value_of(gate[at]);
      held[j] = value(at, gates[j]);
    }
    sum = fmaf(held[j], held[j], sum);
  }
  for (int e = lane + kFinishHeld * lanes; e < length; e += lanes) {
    const int at = column(e);
    const float x = value(at, value_of(gate[at]));
    sum = fmaf(x, x, sum);
  }
  const float scale = 1.0f / sqrtf((kWide ? block_total(sum, shared) : warp_sum(sum)) / float(length) + p.eps);
  auto finish = [&](int at, float x, float z) {
    const float y = x * scale * __bfloat162float(p.norm[at]);
    store_value(out + at, p.gate_first ? y : y * sigmoid_for<T>(z));
  };
#pragma unroll
  for (int j = 0; j < kFinishHeld; ++j) {
    const int e = lane + j * lanes;
    if (e < length) finish(column(e), held[j], gates[j]);
  }
  for (int e = lane + kFinishHeld * lanes; e < length; e += lanes) {
    const int at = column(e);
    const float z = value_of(gate[at]);
    finish(at, value(at, z), z);
  }
  if (group == 0) {
    if (!packed)
      for (int at = lane; at < width; at += lanes)
        if (at % p.vdim_pad >= p.vdim) store_value(out + at, 0.0f);
    for (int at = width + lane; at < p.out_stride; at += lanes) store_value(out + at, 0.0f);
  }
}

template <bool kDelta>
void launch_step_strips(const OuterStateParams& p, cudaStream_t stream, bool pdl) {
  const dim3 grid(unsigned(p.heads), unsigned(p.vdim_pad / 16));
  if (p.dim_pad <= 32) return launch(outer_step_kernel<kDelta, 1>, grid, dim3(128), 0, stream, pdl, p);
  if (p.dim_pad <= 64) return launch(outer_step_kernel<kDelta, 2>, grid, dim3(128), 0, stream, pdl, p);
  if (p.dim_pad <= 128) return launch(outer_step_kernel<kDelta, 4>, grid, dim3(128), 0, stream, pdl, p);
  if (p.dim_pad <= 256) return launch(outer_step_kernel<kDelta, 8>, grid, dim3(128), 0, stream, pdl, p);
  launch(outer_step_kernel<kDelta, 16>, grid, dim3(128), 0, stream, pdl, p);
}

}  // namespace

template <typename T>
void launch_outer_prepare(const OuterStateParams& p, cudaStream_t stream, bool pdl) {
  if (p.rows < 1 || p.rows > kPendingRows) throw std::invalid_argument("a state step takes 1..16 rows");
  const int warps = p.rows * (2 * p.key_heads + p.heads + (p.delta ? p.heads : (p.heads + 31) / 32));
  const dim3 grid(unsigned((warps + 3) / 4));
  if (p.taps == 2) return launch(outer_prepare_kernel<T, 2>, grid, dim3(128), 0, stream, pdl, p);
  if (p.taps == 3) return launch(outer_prepare_kernel<T, 3>, grid, dim3(128), 0, stream, pdl, p);
  if (p.taps == 4) return launch(outer_prepare_kernel<T, 4>, grid, dim3(128), 0, stream, pdl, p);
  launch(outer_prepare_kernel<T, 0>, grid, dim3(128), 0, stream, pdl, p);
}
void launch_outer_conv(const OuterStateParams& p, bf16* out, float* inverse, cudaStream_t stream, bool pdl) {
  const int warps = (p.rows + kConvRows - 1) / kConvRows * (2 * p.key_heads + p.heads);
  const dim3 grid(unsigned((warps + 3) / 4));
  if (p.taps == 2) return launch(outer_conv_kernel<2>, grid, dim3(128), 0, stream, pdl, p, out, inverse);
  if (p.taps == 3) return launch(outer_conv_kernel<3>, grid, dim3(128), 0, stream, pdl, p, out, inverse);
  if (p.taps == 4) return launch(outer_conv_kernel<4>, grid, dim3(128), 0, stream, pdl, p, out, inverse);
  launch(outer_conv_kernel<0>, grid, dim3(128), 0, stream, pdl, p, out, inverse);
}
void launch_outer_step(const OuterStateParams& p, cudaStream_t stream, bool pdl) {
  if (p.rows < 1 || p.rows > kPendingRows || p.dim_pad > kMaxHeadDim)
    throw std::invalid_argument("a state step takes 1..16 rows and key sizes up to 512");
  p.delta ? launch_step_strips<true>(p, stream, pdl) : launch_step_strips<false>(p, stream, pdl);
}
template <typename T>
void launch_state_finish(const StateFinishParams& p, cudaStream_t stream, bool pdl) {
  const int items = p.rows * p.groups + p.tail_rows * ((p.channels + kTailPiece - 1) / kTailPiece), length = p.heads * p.vdim / p.groups;
  if (length > 512)
    launch(state_finish_kernel<T, true>, dim3(unsigned(items)), dim3(256), 0, stream, pdl, p);
  else
    launch(state_finish_kernel<T, false>, dim3(unsigned((items + 3) / 4)), dim3(128), 0, stream, pdl, p);
}
template void launch_outer_prepare<bf16>(const OuterStateParams&, cudaStream_t, bool);
template void launch_outer_prepare<float>(const OuterStateParams&, cudaStream_t, bool);
template void launch_state_finish<bf16>(const StateFinishParams&, cudaStream_t, bool);
template void launch_state_finish<float>(const StateFinishParams&, cudaStream_t, bool);

}  // namespace ei
