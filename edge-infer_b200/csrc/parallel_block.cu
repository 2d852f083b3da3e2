// Blocks whose mixer and feed-forward read the same stream: the embedding (with its pair table) and the join that adds
// both scaled results and leaves the layer norms the next block starts from. One block of threads per row.
#include "layered_device.cuh"

#include <algorithm>

namespace ei {
namespace {

constexpr int kHeld = 4;  // quads of a row a thread keeps in registers; the rest is read again
constexpr int kMostThreads = 1024;

__device__ __forceinline__ float masked_sum(float4 x, int i, int width) {
  return (i < width ? x.x : 0.0f) + (i + 1 < width ? x.y : 0.0f) + (i + 2 < width ? x.z : 0.0f) + (i + 3 < width ? x.w : 0.0f);
}
__device__ __forceinline__ float masked_squares(float4 x, float mean, int i, int width) {
  const float a = x.x - mean, b = x.y - mean, c = x.z - mean, d = x.w - mean;
  return (i < width ? a * a : 0.0f) + (i + 1 < width ? b * b : 0.0f) + (i + 2 < width ? c * c : 0.0f) + (i + 3 < width ? d * d : 0.0f);
}
__device__ __forceinline__ float4 weighted(float4 x, float mean, float scale, float4 w) {
  return make_float4((x.x - mean) * scale * w.x, (x.y - mean) * scale * w.y, (x.z - mean) * scale * w.z, (x.w - mean) * scale * w.w);
}

// The normed rows of a row whose quads are in `held` (and in `residual`, written by the same threads). `columns`: its
// stride in the residual; the weights are zero beyond the width. `ahead`: both weights of a thread's first quad.
struct FirstWeights {
  float4 first, second;
};
__device__ __forceinline__ FirstWeights first_weights(const RowNorms& n, int columns) {
  const int i = threadIdx.x * 4;
  const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  return {i < columns ? load_quad(n.first + i) : zero, i < columns && n.second ? load_quad(n.second + i) : zero};
}
template <typename T>
__device__ __forceinline__ void norm_row(const RowNorms& n, const float4 (&held)[kHeld], const float* residual, int columns,
                                         int row, float* shared, const FirstWeights& ahead) {
  const int step = blockDim.x * 4;
  float sum = 0.0f;
#pragma unroll
  for (int j = 0; j < kHeld; ++j) sum += masked_sum(held[j], threadIdx.x * 4 + j * step, n.width);
  for (int i = threadIdx.x * 4 + kHeld * step; i < columns; i += step)
    sum += masked_sum(*reinterpret_cast<const float4*>(residual + i), i, n.width);
  const float mean = block_total(sum, shared) / float(n.width);
  float squares = 0.0f;
#pragma unroll
  for (int j = 0; j < kHeld; ++j) squares += masked_squares(held[j], mean, threadIdx.x * 4 + j * step, n.width);
  for (int i = threadIdx.x * 4 + kHeld * step; i < columns; i += step)
    squares += masked_squares(*reinterpret_cast<const float4*>(residual + i), mean, i, n.width);
  const float scale = 1.0f / sqrtf(block_total(squares, shared + kMostThreads / 32) / float(n.width) + n.eps);
  T* first = static_cast<T*>(n.normed_first) + size_t(row) * n.stride;
  T* second = n.second ? static_cast<T*>(n.normed_second) + size_t(row) * n.stride : nullptr;
  const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  auto emit = [&](int i, float4 x) {
    const bool live = i < columns, held_ahead = i == int(threadIdx.x) * 4;
    store_quad(first + i, live ? weighted(x, mean, scale, held_ahead ? ahead.first : load_quad(n.first + i)) : zero);
    if (second) store_quad(second + i, live ? weighted(x, mean, scale, held_ahead ? ahead.second : load_quad(n.second + i)) : zero);
  };
#pragma unroll
  for (int j = 0; j < kHeld; ++j) {
    const int i = threadIdx.x * 4 + j * step;
    if (i < n.stride) emit(i, held[j]);
  }
  for (int i = threadIdx.x * 4 + kHeld * step; i < n.stride; i += step)
    emit(i, i < columns ? *reinterpret_cast<const float4*>(residual + i) : zero);
}

template <typename T>
__global__ void __launch_bounds__(kMostThreads) parallel_embed_kernel(const ParallelEmbedParams p) {
  __shared__ uint32_t token_shared;
  __shared__ unsigned long long pair_shared;
  __shared__ float shared[2 * kMostThreads / 32];
  const FirstWeights ahead = first_weights(p.norms, p.residual_stride);
  grid_dependency_wait();
  const int row = blockIdx.x;
  if (threadIdx.x == 0) {
    token_shared = take_step_token(p.token, row);
    if (p.pairs.table) {
      const int context = p.token.control->context, position = context + row;
      unsigned long long pick = p.pairs.buckets;
      if (row > 0 || context > 0) {
        const uint32_t previous = row > 0 ? step_token_of(p.token, p.token.control, row - 1, row - 1)
                                          : p.pairs.history[min(context, p.token.capacity) - 1];
        pick = (previous * p.pairs.mul_prev + token_shared * p.pairs.mul_cur) % p.pairs.buckets;
      }
      pair_shared = pick;
      if (context >= 0 && context + p.token.rows <= p.token.capacity) p.pairs.history[position] = token_shared;
    }
  }
  __syncthreads();
  grid_launch_dependents();
  const uint32_t token = token_shared < uint32_t(p.token.vocab) ? token_shared : 0u;
  const bf16* own = p.table + size_t(token) * p.table_stride;
  const bf16* pair = p.pairs.table ? p.pairs.table + size_t(pair_shared) * p.pairs.stride : nullptr;
  float* residual = p.residual + size_t(row) * p.residual_stride;
  float4 held[kHeld];
  auto fetch = [&](int i) {
    float4 x = load_quad(own + i);
    if (pair) x = add(x, load_quad(pair + i));
    *reinterpret_cast<float4*>(residual + i) = x;
    return x;
  };
#pragma unroll
  for (int j = 0; j < kHeld; ++j) {
    const int i = (threadIdx.x + j * blockDim.x) * 4;
    held[j] = i < p.residual_stride ? fetch(i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  }
  for (int i = (threadIdx.x + kHeld * blockDim.x) * 4; i < p.residual_stride; i += blockDim.x * 4) fetch(i);
  norm_row<T>(p.norms, held, residual, p.residual_stride, row, shared, ahead);
}

template <typename T>
__global__ void __launch_bounds__(kMostThreads) parallel_join_kernel(const ParallelJoinParams p) {
  __shared__ float shared[2 * kMostThreads / 32];
  // Weights do not come from the preceding kernel.
  const FirstWeights ahead = first_weights(p.norms, p.residual_stride);
  const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  const bool live = int(threadIdx.x) * 4 < p.residual_stride;
  const float4 mixed_ahead = live ? load_quad(p.mixed_scale + threadIdx.x * 4) : zero;
  const float4 fed_ahead = live && p.fed ? load_quad(p.fed_scale + threadIdx.x * 4) : zero;
  grid_dependency_wait();
  grid_launch_dependents();
  const int row = blockIdx.x;
  float* residual = p.residual + size_t(row) * p.residual_stride;
  const size_t slice = size_t(p.rows) * p.residual_stride, at = size_t(row) * p.residual_stride;
  auto total = [&](const float* partial, int ksplit, int i) {
    float4 y = *reinterpret_cast<const float4*>(partial + at + i);
    for (int s = 1; s < ksplit; ++s) y = add(y, *reinterpret_cast<const float4*>(partial + s * slice + at + i));
    return y;
  };
  auto join = [&](int i) {
    float4 x = *reinterpret_cast<const float4*>(residual + i);
    const bool held_ahead = i == int(threadIdx.x) * 4;
    float4 y = total(p.mixed, p.mixed_ksplit, i), s = held_ahead ? mixed_ahead : load_quad(p.mixed_scale + i);
    y = make_float4(y.x * s.x, y.y * s.y, y.z * s.z, y.w * s.w);
    if (p.fed) {
      const float4 f = total(p.fed, p.fed_ksplit, i);
      s = held_ahead ? fed_ahead : load_quad(p.fed_scale + i);
      y = make_float4(fmaf(f.x, s.x, y.x), fmaf(f.y, s.y, y.y), fmaf(f.z, s.z, y.z), fmaf(f.w, s.w, y.w));
    }
    x = add(x, y);
    *reinterpret_cast<float4*>(residual + i) = x;
    if (p.tap) {
      float* tap = p.tap + size_t(row) * p.tap_width;
      const float values[4] = {x.x, x.y, x.z, x.w};
      for (int j = 0; j < 4; ++j)
        if (i + j < p.tap_width) tap[i + j] = values[j];
    }
    return x;
  };
  float4 held[kHeld];
#pragma unroll
  for (int j = 0; j < kHeld; ++j) {
    const int i = (threadIdx.x + j * blockDim.x) * 4;
    held[j] = i < p.residual_stride ? join(i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  }
  for (int i = (threadIdx.x + kHeld * blockDim.x) * 4; i < p.residual_stride; i += blockDim.x * 4) join(i);
  norm_row<T>(p.norms, held, residual, p.residual_stride, row, shared, ahead);
}

// A few rows: one quad per thread as far as a block goes. Many: blocks of 256.
unsigned row_threads(int rows, int stride) {
  const int whole = (stride / 4 + 31) / 32 * 32;
  return unsigned(std::min(whole, rows <= kMaxRows ? kMostThreads : 256));
}

}  // namespace

template <typename T>
void launch_parallel_embed(const ParallelEmbedParams& p, cudaStream_t stream, bool pdl) {
  launch(parallel_embed_kernel<T>, dim3(unsigned(p.token.rows)), dim3(row_threads(p.token.rows, p.norms.stride)), 0, stream, pdl, p);
}
template <typename T>
void launch_parallel_join(const ParallelJoinParams& p, cudaStream_t stream, bool pdl) {
  launch(parallel_join_kernel<T>, dim3(unsigned(p.rows)), dim3(row_threads(p.rows, p.norms.stride)), 0, stream, pdl, p);
}
template void launch_parallel_embed<bf16>(const ParallelEmbedParams&, cudaStream_t, bool);
template void launch_parallel_embed<float>(const ParallelEmbedParams&, cudaStream_t, bool);
template void launch_parallel_join<bf16>(const ParallelJoinParams&, cudaStream_t, bool);
template void launch_parallel_join<float>(const ParallelJoinParams&, cudaStream_t, bool);

}  // namespace ei
