// Causal grouped-query attention with free head sizes: query / key size and value size may differ, both up to 256 in
// steps of 16 for the tiled kernels, the score scale and a per-head softmax sink are parameters, and the softmax
// weights keep 16 significant bits in the product with the values (each weight is split into two BF16 terms).
//
// The tile loop is that of the 128-wide verify attention (attention.cu): K and V tiles of 64 tokens by TMA through a
// ring of two or three stages on mbarriers with bounded block-uniform waits, scores and running sums in FP32, mma.sync on
// ldmatrix fragments. What differs:
//  * a staged tile is [piece of a head row][token][up to 128 B]; a head row of `pad` values is cut into pieces of 64,
//    32 or 16 values, whichever divides it, each with the TMA swizzle of its width (128 / 64 / 32 bytes), so the
//    cache needs no padding beyond a multiple of 16;
//  * query rows of all heads of a KV group are stacked over the whole row range and dealt to blocks of up to four
//    warps, 16 stacked rows per warp, so any group size and row count works;
//  * kernels are compiled for sizes up to 64, 128 and 256, and for keys up to 256 with values up to 128, with the sizes
//    known at compile time when they are exactly 64, 128 or 192 and 128;
//  * a key may end in a part that all heads share (latent attention's rotated key), fetched from a tensor of its own;
//  * the finished output may pass a sigmoid gate.
#include "layered_device.cuh"

#include <algorithm>
#include <stdexcept>

namespace ei {
namespace {

constexpr int kTile = 64;
constexpr int kMostStages = 3;
// Tiles in flight: two where three would keep a second block off the SM.
constexpr int stages_for(int keys, int values) { return keys + values > 256 ? 2 : kMostStages; }
constexpr int kMaxWarps = 4;

struct SizedShared {
  uint64_t full[kMostStages];
  int failed;
};

// Byte offset of (token, 16-byte piece of the head row) in a staged tile whose boxes are 2^shift pieces wide.
__device__ __forceinline__ int staged_offset(int token, int piece, int shift) {
  const int pitch = 16 << shift;
  const int at = (piece >> shift) * (kTile * pitch) + token * pitch + ((piece & ((1 << shift) - 1)) << 4);
  return at ^ (((at >> 7) & ((1 << shift) - 1)) << 4);
}

size_t sized_shared_bytes(int stages, int dim_pad, int vdim_pad) {
  return size_t(stages) * kTile * (dim_pad + vdim_pad) * 2 + 1024 + 64;
}

// kDirect = false: block (kv head, split of the sequence, part of the stacked rows) writes (o, m, l) partials.
// kDirect = true: block (kv head, part) covers its rows' whole history and writes the finished output; parts with the
// longest histories start first.
template <int kKeys, int kValues, bool kExact, bool kDirect>
__global__ void __launch_bounds__(kMaxWarps * 32) sized_attention_kernel(const __grid_constant__ SizedAttentionParams p) {
  extern __shared__ unsigned char sized_smem_raw[];
  unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(sized_smem_raw) + 1023) &
                                                         ~uintptr_t(1023));
  constexpr int kSteps = kKeys / 16, kTiles = kValues / 8, kStages = stages_for(kKeys, kValues);
  const int dim = kExact ? kKeys : p.dim_pad, vdim = kExact ? kValues : p.vdim_pad;
  const int k_steps = dim / 16, v_tiles = vdim / 8;
  const int k_shift = kExact ? 3 : p.k_shift, v_shift = kExact ? 3 : p.v_shift;
  const int k_bytes = kTile * dim * 2, v_bytes = kTile * vdim * 2, stage_bytes = k_bytes + v_bytes;
  SizedShared* sh = reinterpret_cast<SizedShared*>(smem + size_t(kStages) * stage_bytes);

  const int offset = *p.device_offset;
  const int kv_head = blockIdx.x;
  if (offset < 0 || offset + p.rows > p.capacity) {
    grid_dependency_wait();
    return;
  }
  const int group = p.heads / p.kv_heads;
  const int warps = blockDim.x >> 5;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
  const int stacked = p.rows * group;
  const int part = kDirect ? int(gridDim.y) - 1 - int(blockIdx.y) : int(blockIdx.z);
  const int first_stacked = part * warps * 16;
  const int last_row = min(stacked - 1, first_stacked + warps * 16 - 1) / group;
  const int split = kDirect ? 0 : blockIdx.y;
  const int start = kDirect ? 0 : split * p.chunk;
  const int length = offset + last_row + 1;          // tokens this block's rows may see
  if (start >= offset + p.rows) return;              // beyond every row: no other block's work depends on this one
  const int end = kDirect ? length : min(start + p.chunk, length);
  const int tiles = max(0, (end - start + kTile - 1) / kTile);
  const uint32_t wait_limit = p.wait_limit ? p.wait_limit : kTmaWaitLimit;

  if (threadIdx.x == 0) {
    for (int s = 0; s < kStages; ++s) mbarrier_init(&sh->full[s], 1);
    sh->failed = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  __syncthreads();
  auto request = [&](int tile) {
    const int stage = tile % kStages;
    unsigned char* base = smem + size_t(stage) * stage_bytes;
    mbarrier_expect_tx(&sh->full[stage], uint32_t(stage_bytes) + (tile == 0 ? p.fault_tx : 0u));
    tma_load_4d(base, &p.k_map, 0, start + tile * kTile, 0, kv_head, &sh->full[stage]);
    if (p.shared_pad)
      tma_load_4d(base + kTile * (dim - p.shared_pad) * 2, &p.shared_map, 0, start + tile * kTile, 0, 0, &sh->full[stage]);
    tma_load_4d(base + k_bytes, &p.v_map, 0, start + tile * kTile, 0, kv_head, &sh->full[stage]);
  };
  const bool settled = end <= offset && !p.fresh;  // nothing in this chunk is written by the preceding kernel
  if (!settled) grid_dependency_wait();
  if (threadIdx.x == 0)
    for (int tile = 0; tile < min(kStages, tiles); ++tile) request(tile);
  if (settled) grid_dependency_wait();
  grid_launch_dependents();

  // Stacked row i = row * group + head of the group.
  const int i_lo = first_stacked + warp * 16 + g, i_hi = i_lo + 8;
  const bool live_lo = i_lo < stacked, live_hi = i_hi < stacked;
  const int r_lo = live_lo ? i_lo / group : 0, r_hi = live_hi ? i_hi / group : 0;
  const int h_lo = kv_head * group + (live_lo ? i_lo % group : 0);
  const int h_hi = kv_head * group + (live_hi ? i_hi % group : 0);
  uint32_t qa[kSteps][4];
  {
    const bf16* q_lo = static_cast<const bf16*>(p.q) + size_t(r_lo) * p.q_stride + size_t(h_lo) * dim;
    const bf16* q_hi = static_cast<const bf16*>(p.q) + size_t(r_hi) * p.q_stride + size_t(h_hi) * dim;
#pragma unroll
    for (int kk = 0; kk < kSteps; ++kk) {
      const bool on = kExact || kk < k_steps;
      qa[kk][0] = on && live_lo ? *reinterpret_cast<const uint32_t*>(q_lo + kk * 16 + 2 * c) : 0u;
      qa[kk][1] = on && live_hi ? *reinterpret_cast<const uint32_t*>(q_hi + kk * 16 + 2 * c) : 0u;
      qa[kk][2] = on && live_lo ? *reinterpret_cast<const uint32_t*>(q_lo + kk * 16 + 8 + 2 * c) : 0u;
      qa[kk][3] = on && live_hi ? *reinterpret_cast<const uint32_t*>(q_hi + kk * 16 + 8 + 2 * c) : 0u;
    }
  }
  const int limit_lo = offset + r_lo, limit_hi = offset + r_hi;  // last visible token of each row
  // The last token any row of this warp sees: whole tiles beyond it are skipped by the warp.
  const int warp_first = first_stacked + warp * 16;
  const int warp_limit = warp_first < stacked ? offset + min(stacked - 1, warp_first + 15) / group : -1;

  float o[kTiles][4];
#pragma unroll
  for (int d = 0; d < kTiles; ++d) o[d][0] = o[d][1] = o[d][2] = o[d][3] = 0.0f;
  float m_lo = -INFINITY, m_hi = -INFINITY, l_lo = 0.0f, l_hi = 0.0f;

  int tile = 0;
  bool gave_up = false;
  for (; tile < tiles; ++tile) {
    const int stage = tile % kStages;
    if (!mbarrier_wait(&sh->full[stage], (tile / kStages) & 1, wait_limit)) sh->failed = 1;
    unsigned char* ks = smem + size_t(stage) * stage_bytes;
    unsigned char* vs = ks + k_bytes;
    const int first = start + tile * kTile;
    if (end - first < kTile) {
      // Rows of the last tile beyond the block's history hold whatever the cache holds there; their scores are masked
      // and their values cleared, so that a non-finite leftover cannot pass through a zero weight.
      const int live = end - first, pieces = vdim / 8;
      for (int i = threadIdx.x; i < (kTile - live) * pieces; i += blockDim.x)
        *reinterpret_cast<uint4*>(vs + staged_offset(live + i / pieces, i % pieces, v_shift)) = make_uint4(0, 0, 0, 0);
      __syncthreads();
    }
    if (first <= warp_limit) {
      float s[8][4];
#pragma unroll
      for (int j = 0; j < 8; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.0f;
      // One ldmatrix.x4 brings the fragments of one k-step for two tiles of eight tokens.
#pragma unroll
      for (int kk = 0; kk < kSteps; ++kk) {
        if (kExact || kk < k_steps) {
#pragma unroll
          for (int j = 0; j < 8; j += 2) {
            uint32_t b0, b1, b2, b3;
            ldmatrix_x4(b0, b1, b2, b3,
                        ks + staged_offset((j + (lane >> 4)) * 8 + (lane & 7), 2 * kk + ((lane >> 3) & 1), k_shift));
            mma_bf16_16816(s[j], qa[kk][0], qa[kk][1], qa[kk][2], qa[kk][3], b0, b1);
            mma_bf16_16816(s[j + 1], qa[kk][0], qa[kk][1], qa[kk][2], qa[kk][3], b2, b3);
          }
        }
      }
      float tile_max_lo = -INFINITY, tile_max_hi = -INFINITY;
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int t0 = first + j * 8 + 2 * c, t1 = t0 + 1;
        s[j][0] = t0 <= limit_lo ? s[j][0] * p.scale : -INFINITY;
        s[j][1] = t1 <= limit_lo ? s[j][1] * p.scale : -INFINITY;
        s[j][2] = t0 <= limit_hi ? s[j][2] * p.scale : -INFINITY;
        s[j][3] = t1 <= limit_hi ? s[j][3] * p.scale : -INFINITY;
        tile_max_lo = fmaxf(tile_max_lo, fmaxf(s[j][0], s[j][1]));
        tile_max_hi = fmaxf(tile_max_hi, fmaxf(s[j][2], s[j][3]));
      }
      tile_max_lo = fmaxf(tile_max_lo, __shfl_xor_sync(0xffffffffu, tile_max_lo, 1));
      tile_max_lo = fmaxf(tile_max_lo, __shfl_xor_sync(0xffffffffu, tile_max_lo, 2));
      tile_max_hi = fmaxf(tile_max_hi, __shfl_xor_sync(0xffffffffu, tile_max_hi, 1));
      tile_max_hi = fmaxf(tile_max_hi, __shfl_xor_sync(0xffffffffu, tile_max_hi, 2));
      const float new_lo = fmaxf(m_lo, tile_max_lo), new_hi = fmaxf(m_hi, tile_max_hi);
      const float base_lo = new_lo == -INFINITY ? 0.0f : new_lo;  // nothing visible yet: exp() gives 0
      const float base_hi = new_hi == -INFINITY ? 0.0f : new_hi;
      const float rescale_lo = __expf(m_lo - base_lo), rescale_hi = __expf(m_hi - base_hi);
      m_lo = new_lo;
      m_hi = new_hi;
      float sum_lo = 0.0f, sum_hi = 0.0f;
      uint32_t pa[8][2], pr[8][2];  // the weights' leading BF16 terms and what those leave
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float p0 = __expf(s[j][0] - base_lo), p1 = __expf(s[j][1] - base_lo);
        const float p2 = __expf(s[j][2] - base_hi), p3 = __expf(s[j][3] - base_hi);
        sum_lo += p0 + p1;
        sum_hi += p2 + p3;
        pa[j][0] = pack_bf16(p0, p1);
        pa[j][1] = pack_bf16(p2, p3);
        pr[j][0] = pack_bf16(p0 - bf16_lo(pa[j][0]), p1 - bf16_hi(pa[j][0]));
        pr[j][1] = pack_bf16(p2 - bf16_lo(pa[j][1]), p3 - bf16_hi(pa[j][1]));
      }
      l_lo = l_lo * rescale_lo + sum_lo;
      l_hi = l_hi * rescale_hi + sum_hi;
#pragma unroll
      for (int d = 0; d < kTiles; ++d) {
        o[d][0] *= rescale_lo;
        o[d][1] *= rescale_lo;
        o[d][2] *= rescale_hi;
        o[d][3] *= rescale_hi;
      }
#pragma unroll
      for (int t = 0; t < 4; ++t) {
#pragma unroll
        for (int d = 0; d < kTiles; d += 2) {
          if (kExact || d < v_tiles) {
            uint32_t b0, b1, b2, b3;
            ldmatrix_x4_trans(b0, b1, b2, b3,
                              vs + staged_offset(t * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), d + (lane >> 4), v_shift));
            mma_bf16_16816(o[d], pa[2 * t][0], pa[2 * t][1], pa[2 * t + 1][0], pa[2 * t + 1][1], b0, b1);
            mma_bf16_16816(o[d + 1], pa[2 * t][0], pa[2 * t][1], pa[2 * t + 1][0], pa[2 * t + 1][1], b2, b3);
            mma_bf16_16816(o[d], pr[2 * t][0], pr[2 * t][1], pr[2 * t + 1][0], pr[2 * t + 1][1], b0, b1);
            mma_bf16_16816(o[d + 1], pr[2 * t][0], pr[2 * t][1], pr[2 * t + 1][0], pr[2 * t + 1][1], b2, b3);
          }
        }
      }
    }
    __syncthreads();  // every warp is done with this stage
    gave_up = sh->failed != 0;
    if (gave_up) break;
    if (threadIdx.x == 0 && tile + kStages < tiles) request(tile + kStages);
  }
  if (gave_up) {
    if (threadIdx.x == 0) {
      for (int t = max(tile, p.fault_tx ? 1 : 0); t < min(tile + kStages, tiles); ++t)
        mbarrier_wait(&sh->full[t % kStages], (t / kStages) & 1, wait_limit);
      if (p.status) atomicOr(p.status, 4);
    }
    return;
  }
  l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1);
  l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
  l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1);
  l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);

  if (kDirect) {
    auto finish = [&](float m, float l, int head) {
      if (!p.sink) return l > 0.0f ? p.out_scale / l : 0.0f;
      const float sink = p.sink[head], top = fmaxf(m, sink);
      const float own = __expf(m - top);
      return p.out_scale * own / (l * own + __expf(sink - top));
    };
    const float f_lo = finish(m_lo, l_lo, h_lo), f_hi = finish(m_hi, l_hi, h_hi);
    bf16* out = static_cast<bf16*>(p.out);
    bf16* d_lo = out + size_t(r_lo) * p.out_stride + size_t(h_lo) * vdim;
    bf16* d_hi = out + size_t(r_hi) * p.out_stride + size_t(h_hi) * vdim;
    const bf16* gate = static_cast<const bf16*>(p.gate);
    const bf16* g_lo = gate ? gate + size_t(r_lo) * p.gate_stride + size_t(h_lo) * vdim : nullptr;
    const bf16* g_hi = gate ? gate + size_t(r_hi) * p.gate_stride + size_t(h_hi) * vdim : nullptr;
    auto gated = [&](const bf16* g, int at, float a, float b) {
      if (!gate) return pack_bf16(a, b);
      const float2 z = load_pair(g + at);
      return pack_bf16(a * quick_sigmoid(z.x), b * quick_sigmoid(z.y));
    };
#pragma unroll
    for (int d = 0; d < kTiles; ++d) {
      if (kExact || d < v_tiles) {
        const int at = d * 8 + 2 * c;
        if (live_lo) *reinterpret_cast<uint32_t*>(d_lo + at) = gated(g_lo, at, o[d][0] * f_lo, o[d][1] * f_lo);
        if (live_hi) *reinterpret_cast<uint32_t*>(d_hi + at) = gated(g_hi, at, o[d][2] * f_hi, o[d][3] * f_hi);
      }
    }
    return;
  }
  const size_t slots = size_t(p.rows) * p.heads;
  const int pitch = vdim + 4;
  float* d_lo = p.scratch + (size_t(split) * slots + size_t(r_lo) * p.heads + h_lo) * pitch;
  float* d_hi = p.scratch + (size_t(split) * slots + size_t(r_hi) * p.heads + h_hi) * pitch;
#pragma unroll
  for (int d = 0; d < kTiles; ++d) {
    if (kExact || d < v_tiles) {
      if (live_lo) *reinterpret_cast<float2*>(d_lo + d * 8 + 2 * c) = make_float2(o[d][0], o[d][1]);
      if (live_hi) *reinterpret_cast<float2*>(d_hi + d * 8 + 2 * c) = make_float2(o[d][2], o[d][3]);
    }
  }
  if (c == 0) {
    if (live_lo) {
      d_lo[vdim] = m_lo;
      d_lo[vdim + 1] = l_lo;
    }
    if (live_hi) {
      d_hi[vdim] = m_hi;
      d_hi[vdim + 1] = l_hi;
    }
  }
}

// Any head size, FP32 arithmetic: one block per (row, head), a lane scores one key of a warp's 32 and the warp's lanes
// share the value columns, kColumns each; the four warps' running sums meet in shared memory.
template <typename T, int kColumns>
__global__ void __launch_bounds__(128) plain_attention_kernel(const SizedAttentionParams p) {
  extern __shared__ float plain_smem[];
  float* query = plain_smem;                       // [dim_pad]
  float* sums = plain_smem + p.dim_pad;            // [4][vdim_pad]
  __shared__ float tops[4], denominators[4];
  grid_dependency_wait();
  grid_launch_dependents();
  const int offset = *p.device_offset;
  if (offset < 0 || offset + p.rows > p.capacity) return;
  const int row = blockIdx.x / p.heads, head = blockIdx.x - row * p.heads;
  const int kv_head = head / (p.heads / p.kv_heads);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int length = offset + row + 1;
  const T* q = static_cast<const T*>(p.q) + size_t(row) * p.q_stride + size_t(head) * p.dim_pad;
  for (int i = threadIdx.x; i < p.dim_pad; i += blockDim.x) query[i] = value_of(q[i]);
  __syncthreads();
  const T* keys = static_cast<const T*>(p.k) + size_t(kv_head) * p.dim_pad;
  const T* values = static_cast<const T*>(p.v) + size_t(kv_head) * p.vdim_pad;
  float acc[kColumns];
#pragma unroll
  for (int j = 0; j < kColumns; ++j) acc[j] = 0.0f;
  float top = -INFINITY, denominator = 0.0f;
  for (int first = warp * 32; first < length; first += 128) {
    const int key = first + lane;
    float score = -INFINITY;
    if (key < length) {
      const T* k = keys + size_t(key) * p.k_stride;
      float sum = 0.0f;
      for (int i = 0; i < p.dim_pad; ++i) sum = fmaf(query[i], value_of(k[i]), sum);
      score = sum * p.scale;
    }
    const float new_top = fmaxf(top, warp_max(score));  // finite: the warp's first key is live
    const float rescale = expf(top - new_top), weight = expf(score - new_top);
    top = new_top;
    denominator = denominator * rescale + warp_sum(weight);
#pragma unroll
    for (int j = 0; j < kColumns; ++j) acc[j] *= rescale;
    const int live = min(32, length - first);
    for (int t = 0; t < live; ++t) {
      const float w = __shfl_sync(0xffffffffu, weight, t);
      const T* v = values + size_t(first + t) * p.v_stride;
#pragma unroll
      for (int j = 0; j < kColumns; ++j)
        if (lane + 32 * j < p.vdim_pad) acc[j] = fmaf(w, value_of(v[lane + 32 * j]), acc[j]);
    }
  }
#pragma unroll
  for (int j = 0; j < kColumns; ++j)
    if (lane + 32 * j < p.vdim_pad) sums[warp * p.vdim_pad + lane + 32 * j] = acc[j];
  if (lane == 0) {
    tops[warp] = top;
    denominators[warp] = denominator;
  }
  __syncthreads();
  float all = p.sink ? p.sink[head] : -INFINITY;
  for (int w = 0; w < 4; ++w) all = fmaxf(all, tops[w]);
  float total = p.sink ? expf(p.sink[head] - all) : 0.0f, weights[4];
#pragma unroll
  for (int w = 0; w < 4; ++w) {
    weights[w] = tops[w] == -INFINITY ? 0.0f : expf(tops[w] - all);
    total += denominators[w] * weights[w];
  }
  T* out = static_cast<T*>(p.out) + size_t(row) * p.out_stride + size_t(head) * p.vdim_pad;
  for (int i = threadIdx.x; i < p.vdim_pad; i += blockDim.x) {
    float sum = 0.0f;
#pragma unroll
    for (int w = 0; w < 4; ++w) sum += sums[w * p.vdim_pad + i] * weights[w];
    store_value(out + i, sum / total * p.out_scale);
  }
}

// 16-byte pieces per box row (as log2): the widest of 64, 32 and 16 values that divides the padded head.
int box_shift(int pad) { return pad % 64 == 0 ? 3 : pad % 32 == 0 ? 2 : 1; }

void encode_head_map(CUtensorMap* map, const void* base, int tokens, int token_stride, int kv_heads, int pad, int shift) {
  const int values = 8 << shift;
  const cuuint64_t dims[4] = {cuuint64_t(values), cuuint64_t(tokens), cuuint64_t(pad / values), cuuint64_t(kv_heads)};
  const cuuint64_t strides[3] = {cuuint64_t(token_stride) * 2, cuuint64_t(values) * 2, cuuint64_t(pad) * 2};
  const cuuint32_t box[4] = {cuuint32_t(values), cuuint32_t(kTile), cuuint32_t(pad / values), 1};
  encode_map(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, base, dims, strides, box,
             shift == 3 ? CU_TENSOR_MAP_SWIZZLE_128B : shift == 2 ? CU_TENSOR_MAP_SWIZZLE_64B : CU_TENSOR_MAP_SWIZZLE_32B,
             "sized K / V cache");
}

template <int kKeys, int kValues, bool kExact>
void launch_bucket(const SizedAttentionParams& p, bool direct, cudaStream_t stream, bool pdl) {
  static thread_local int configured_device = -1;
  int device = 0;
  EI_CUDA(cudaGetDevice(&device));
  if (configured_device != device) {
    const int bytes = int(sized_shared_bytes(stages_for(kKeys, kValues), kKeys, kValues));
    EI_CUDA(cudaFuncSetAttribute(sized_attention_kernel<kKeys, kValues, kExact, false>,
                                 cudaFuncAttributeMaxDynamicSharedMemorySize, bytes));
    EI_CUDA(cudaFuncSetAttribute(sized_attention_kernel<kKeys, kValues, kExact, true>,
                                 cudaFuncAttributeMaxDynamicSharedMemorySize, bytes));
    configured_device = device;
  }
  const int stacked = p.rows * (p.heads / p.kv_heads);
  const int warps = std::min(kMaxWarps, (stacked + 15) / 16);
  const unsigned parts = unsigned((stacked + warps * 16 - 1) / (warps * 16));
  const size_t smem = sized_shared_bytes(stages_for(kKeys, kValues), p.dim_pad, p.vdim_pad);
  if (direct)
    launch(sized_attention_kernel<kKeys, kValues, kExact, true>, dim3(p.kv_heads, parts), dim3(warps * 32), smem, stream, pdl, p);
  else
    launch(sized_attention_kernel<kKeys, kValues, kExact, false>, dim3(p.kv_heads, p.max_splits, parts), dim3(warps * 32), smem,
           stream, pdl, p);
}

void launch_sized(const SizedAttentionParams& given, bool direct, cudaStream_t stream, bool pdl) {
  SizedAttentionParams p = given;
  if (!sized_attention_ok(p.dim_pad, p.vdim_pad)) throw std::invalid_argument("tiled attention takes head sizes up to 256");
  const int own = p.dim_pad - p.shared_pad;  // key values of each head's own
  p.k_shift = p.shared_pad ? std::min(box_shift(own), box_shift(p.shared_pad)) : box_shift(own);
  p.v_shift = box_shift(p.vdim_pad);
  // The caches are allocated in whole tiles.
  const int tokens = p.tokens ? p.tokens : (p.capacity + kTile - 1) / kTile * kTile;
  encode_head_map(&p.k_map, p.k, tokens, p.k_stride, p.kv_heads, own, p.k_shift);
  if (p.shared_pad) encode_head_map(&p.shared_map, p.shared, tokens, p.shared_stride, 1, p.shared_pad, p.k_shift);
  encode_head_map(&p.v_map, p.v, tokens, p.v_stride, p.kv_heads, p.vdim_pad, p.v_shift);
  const int widest = std::max(p.dim_pad, p.vdim_pad);
  const bool same = p.dim_pad == p.vdim_pad && p.k_shift == 3;
  if (widest <= 64) {
    if (same && widest == 64) return launch_bucket<64, 64, true>(p, direct, stream, pdl);
    return launch_bucket<64, 64, false>(p, direct, stream, pdl);
  }
  if (widest <= 128) {
    if (same && widest == 128) return launch_bucket<128, 128, true>(p, direct, stream, pdl);
    return launch_bucket<128, 128, false>(p, direct, stream, pdl);
  }
  if (p.vdim_pad <= 128) {
    if (p.dim_pad == 192 && p.vdim_pad == 128 && p.k_shift == 3) return launch_bucket<192, 128, true>(p, direct, stream, pdl);
    return launch_bucket<256, 128, false>(p, direct, stream, pdl);
  }
  return launch_bucket<256, 256, false>(p, direct, stream, pdl);
}

}  // namespace

bool sized_attention_ok(int dim_pad, int vdim_pad) {
  return dim_pad >= 16 && vdim_pad >= 16 && dim_pad % 16 == 0 && vdim_pad % 16 == 0 && dim_pad <= 256 && vdim_pad <= 256;
}

size_t sized_attention_scratch_bytes(size_t rows, size_t heads, size_t vdim_pad, size_t capacity) {
  const size_t chunk = attention_chunk_for(capacity);
  return (capacity + chunk - 1) / chunk * rows * heads * (vdim_pad + 4) * sizeof(float);
}

void launch_sized_attention_step(const SizedAttentionParams& p, cudaStream_t stream, bool pdl) {
  launch_sized(p, false, stream, pdl);
}

void launch_sized_attention_prompt(const SizedAttentionParams& p, cudaStream_t stream, bool pdl) {
  launch_sized(p, true, stream, pdl);
}

template <typename T>
void launch_plain_attention(const SizedAttentionParams& p, cudaStream_t stream, bool pdl) {
  const size_t smem = (size_t(p.dim_pad) + 4 * size_t(p.vdim_pad)) * sizeof(float);
  if (p.vdim_pad > kMaxLatent || smem > 47 * 1024) throw std::invalid_argument("attention head size beyond the supported range");
  const dim3 grid(unsigned(p.rows) * p.heads);
  if (p.vdim_pad <= 512)
    launch(plain_attention_kernel<T, 16>, grid, dim3(128), smem, stream, pdl, p);
  else
    launch(plain_attention_kernel<T, 32>, grid, dim3(128), smem, stream, pdl, p);
}
template void launch_plain_attention<float>(const SizedAttentionParams&, cudaStream_t, bool);
template void launch_plain_attention<bf16>(const SizedAttentionParams&, cudaStream_t, bool);

}  // namespace ei
