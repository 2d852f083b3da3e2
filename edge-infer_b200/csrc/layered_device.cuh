// Device helpers of the kernels of decoders described layer by layer: loads and stores in the activation type, the
// usual nonlinearities, sums over a block.
#pragma once

#include "layered.cuh"

namespace ei {

__device__ __forceinline__ float value_of(bf16 x) { return __bfloat162float(x); }
__device__ __forceinline__ float value_of(float x) { return x; }
__device__ __forceinline__ void store_value(bf16* p, float x) { *p = __float2bfloat16_rn(x); }
__device__ __forceinline__ void store_value(float* p, float x) { *p = x; }
__device__ __forceinline__ float2 load_pair(const bf16* p) {
  const uint32_t v = *reinterpret_cast<const uint32_t*>(p);
  return make_float2(bf16_lo(v), bf16_hi(v));
}
__device__ __forceinline__ float2 load_pair(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ void store_pair(bf16* p, float a, float b) { *reinterpret_cast<uint32_t*>(p) = pack_bf16(a, b); }
__device__ __forceinline__ void store_pair(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ float4 load_quad(const bf16* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  return make_float4(bf16_lo(v.x), bf16_hi(v.x), bf16_lo(v.y), bf16_hi(v.y));
}
__device__ __forceinline__ float4 load_quad(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void store_quad(bf16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
}
__device__ __forceinline__ void store_quad(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }

__device__ __forceinline__ float sigmoid_value(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float silu_exact(float x) { return x / (1.0f + expf(-x)); }
// The fast exponential and quotient (a few units in the last place of FP32) for kernels on BF16 activations.
__device__ __forceinline__ float quick_sigmoid(float x) { return __fdividef(1.0f, 1.0f + __expf(-x)); }
__device__ __forceinline__ float quick_candidate(float u) { return u >= 0.0f ? u + 0.5f : quick_sigmoid(u); }
template <typename T>
__device__ __forceinline__ float sigmoid_for(float x) { return sizeof(T) == 2 ? quick_sigmoid(x) : sigmoid_value(x); }
template <typename T>
__device__ __forceinline__ float silu_for(float x) { return sizeof(T) == 2 ? x * quick_sigmoid(x) : silu_exact(x); }
__device__ __forceinline__ float4 add(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
__device__ __forceinline__ float softplus_value(float x) { return x > 20.0f ? x : log1pf(expf(x)); }
// ln(1 + e^x) with the fast exponential and logarithm: max(x, 0) + ln(1 + y), y = e^-|x|, and for small y the start of
// the logarithm's series, so that no digits are lost to the 1 (relative error below 1e-5).
__device__ __forceinline__ float quick_softplus(float x) {
  const float y = __expf(-fabsf(x));
  const float series = y * fmaf(y, fmaf(y, fmaf(y, fmaf(y, 0.2f, -0.25f), 1.0f / 3.0f), -0.5f), 1.0f);
  return fmaxf(x, 0.0f) + (y < 0.0625f ? series : __logf(1.0f + y));
}

// Sum over the block; `shared` holds a value per warp and is free again after the next block-wide barrier.
__device__ __forceinline__ float block_total(float v, float* shared) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) shared[threadIdx.x >> 5] = v;
  __syncthreads();
  float total = 0.0f;
  for (int w = 0; w < int(blockDim.x >> 5); ++w) total += shared[w];
  return total;
}

// A value as two BF16 terms: the leading one and what it leaves, 16 significant bits together.
__device__ __forceinline__ void split_pair(float a, float b, uint32_t& leading, uint32_t& rest) {
  leading = pack_bf16(a, b);
  rest = pack_bf16(a - bf16_lo(leading), b - bf16_hi(leading));
}

}  // namespace ei
