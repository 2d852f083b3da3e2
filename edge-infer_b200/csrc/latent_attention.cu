// Latent attention: softmax attention whose keys and values are expanded from one latent vector per token, beside a
// rotated key part that all heads share. The cache holds latent and rotated key side by side, one row per token.
//
// A step of at most 16 rows never expands them. A query goes through the key expansion instead (its head's dim values
// become rank values) and scores directly against the cache rows; the softmax-weighted sum of latents goes through the
// value expansion at the end. All heads then read the same rows, so the cache is read once for 16 (row, head) pairs,
// split over blocks along the sequence. The scores and the softmax are FP32; the weights enter the product with the
// latents as two BF16 terms.
//
// A prompt segment expands the keys and values of all cached tokens with the prompt GEMM and runs the tile loop of
// sized_attention.cu over them, with the rotated part fetched from the cache.
#include "layered_device.cuh"

#include <algorithm>
#include <stdexcept>

namespace ei {
namespace {

// Turns the pairs (2 i, 2 i + 1) of `x` and writes them to `to`; values behind them, up to `pad`, are copied. Lanes take
// four values at a time (rotation sizes are even, padded ones multiples of 16).
template <typename T>
__device__ __forceinline__ void turn_quad(const T* x, T* to, const float2* rotation, int dims, int at) {
  float4 v = load_quad(x + at);
  if (at < dims) {
    const float2 t = rotation[at / 2];
    const float a = v.x * t.x - v.y * t.y;
    v.y = v.y * t.x + v.x * t.y;
    v.x = a;
  }
  if (at + 2 < dims) {
    const float2 t = rotation[at / 2 + 1];
    const float a = v.z * t.x - v.w * t.y;
    v.w = v.w * t.x + v.z * t.y;
    v.z = a;
  }
  store_quad(to + at, v);
}

// One warp: latent norm and rotated key of a row into the cache.
template <typename T>
__device__ __forceinline__ void cache_row(const LatentParams& p, int context, int row, int lane) {
  const T* x = static_cast<const T*>(p.fused) + size_t(row) * p.stride + p.latent_at;
  const int position = context + row;
  T* to = static_cast<T*>(p.cache) + size_t(position) * p.row_pad;
  constexpr int kQuads = 4;
  float4 held[kQuads];
  float sum = 0.0f;
  auto square = [&](float4 v) { sum = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, sum)))); };
#pragma unroll
  for (int j = 0; j < kQuads; ++j) {
    const int i = (lane + 32 * j) * 4;
    held[j] = i < p.rank_pad ? load_quad(x + i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  }
#pragma unroll
  for (int j = 0; j < kQuads; ++j) square(held[j]);
  for (int i = (lane + 32 * kQuads) * 4; i < p.rank_pad; i += 128) square(load_quad(x + i));
  const float scale = 1.0f / sqrtf(warp_sum(sum) / float(p.rank) + p.eps);
  auto emit = [&](int i, float4 v) {
    const float4 w = load_quad(p.norm + i);
    store_quad(to + i, make_float4(v.x * scale * w.x, v.y * scale * w.y, v.z * scale * w.z, v.w * scale * w.w));
  };
#pragma unroll
  for (int j = 0; j < kQuads; ++j)
    if ((lane + 32 * j) * 4 < p.rank_pad) emit((lane + 32 * j) * 4, held[j]);
  for (int i = (lane + 32 * kQuads) * 4; i < p.rank_pad; i += 128) emit(i, load_quad(x + i));
  const float2* rotation = p.rotation + size_t(position) * (p.rot_dims / 2);
  for (int i = lane * 4; i < p.rot_pad; i += 128) turn_quad(x + p.rank_pad, to + p.rank_pad, rotation, p.rot_dims, i);
  for (int i = p.rank_pad + p.rot_pad + 4 * lane; i < p.row_pad; i += 128) store_quad(to + i, make_float4(0.0f, 0.0f, 0.0f, 0.0f));
}

// Four values of the rotated part of one head's query, in place or (step form) behind the absorbed query.
template <typename T>
__device__ __forceinline__ void query_quad(const LatentParams& p, bool step, int context, int row, int head, int at) {
  T* q = static_cast<T*>(p.fused) + size_t(row) * p.stride + size_t(head) * (p.dim_pad + p.rot_pad) + p.dim_pad;
  T* to = step ? static_cast<T*>(p.query) + (size_t(row) * p.heads + head) * p.row_pad + p.rank_pad : q;
  if (at < p.rot_pad)
    turn_quad(q, to, p.rotation + size_t(context + row) * (p.rot_dims / 2), p.rot_dims, at);
  else
    store_quad(to + at, make_float4(0.0f, 0.0f, 0.0f, 0.0f));  // a cache row's padding
}

// Blocks [0, absorbing) of a step: 64 latent columns of one head's queries, the sum over the head's dim values of query
// times key expansion, the eight warps taking every eighth value. Then the cache rows, one per warp, then the rotated
// query parts, four values per thread.
constexpr int kPrepareThreads = 256;
constexpr int kAhead = 16;  // rows of the expansion a warp requests before waiting
template <typename T, int kRows>
__global__ void __launch_bounds__(kPrepareThreads) latent_prepare_kernel(const LatentParams p, int absorbing) {
  extern __shared__ __align__(16) unsigned char prepare_smem[];
  float2* parts = reinterpret_cast<float2*>(prepare_smem);                  // [8][rows][32]
  float* query = reinterpret_cast<float*>(parts + size_t(8) * p.rows * 32);  // [rows][dim_pad]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int context = p.control->context;  // written by the previous step
  const bool runs = context >= 0 && context + p.rows <= p.capacity;
  if (int(blockIdx.x) >= absorbing) {
    grid_dependency_wait();
    grid_launch_dependents();
    if (!runs) return;
    const bool step = absorbing > 0;
    const int cache_blocks = (p.rows + 7) / 8, block = blockIdx.x - absorbing;
    if (block < cache_blocks) {
      if (block * 8 + warp < p.rows) cache_row<T>(p, context, block * 8 + warp, lane);
      return;
    }
    const int quads = (step ? p.row_pad - p.rank_pad : p.rot_pad) / 4;
    const int item = (block - cache_blocks) * kPrepareThreads + threadIdx.x, pair = item / quads;
    if (pair < p.rows * p.heads) query_quad<T>(p, step, context, pair / p.heads, pair % p.heads, (item - pair * quads) * 4);
    return;
  }
  const int pieces = p.rank_pad / 64, head = blockIdx.x / pieces, column = (blockIdx.x - head * pieces) * 64 + 2 * lane;
  const bf16* weights = p.expand + size_t(head) * p.dim_pad * p.rank_pad + column;
  float2 held[kAhead];
#pragma unroll
  for (int i = 0; i < kAhead; ++i) {
    const int d = warp + 8 * i;
    held[i] = d < p.dim_pad ? load_pair(weights + size_t(d) * p.rank_pad) : make_float2(0.0f, 0.0f);
  }
  grid_dependency_wait();
  grid_launch_dependents();
  if (!runs) return;
  const T* q = static_cast<const T*>(p.fused) + size_t(head) * (p.dim_pad + p.rot_pad);
  for (int i = threadIdx.x; i < p.rows * p.dim_pad; i += kPrepareThreads)
    query[i] = value_of(q[size_t(i / p.dim_pad) * p.stride + i % p.dim_pad]);
  __syncthreads();
  float2 acc[kRows];
#pragma unroll
  for (int r = 0; r < kRows; ++r) acc[r] = make_float2(0.0f, 0.0f);
  auto absorb = [&](int d, float2 w) {
#pragma unroll
    for (int r = 0; r < kRows; ++r) {
      if (r < p.rows) {
        acc[r].x = fmaf(query[r * p.dim_pad + d], w.x, acc[r].x);
        acc[r].y = fmaf(query[r * p.dim_pad + d], w.y, acc[r].y);
      }
    }
  };
#pragma unroll
  for (int i = 0; i < kAhead; ++i)
    if (warp + 8 * i < p.dim_pad) absorb(warp + 8 * i, held[i]);
  for (int d = warp + 8 * kAhead; d < p.dim_pad; d += 8) absorb(d, load_pair(weights + size_t(d) * p.rank_pad));
#pragma unroll
  for (int r = 0; r < kRows; ++r)
    if (r < p.rows) parts[(warp * p.rows + r) * 32 + lane] = acc[r];
  __syncthreads();
  for (int i = threadIdx.x; i < p.rows * 32; i += kPrepareThreads) {
    const int r = i >> 5;  // lane i & 31 == lane: the block's threads keep their columns
    float2 sum = parts[i];
    for (int w = 1; w < 8; ++w) {
      sum.x += parts[w * p.rows * 32 + i].x;
      sum.y += parts[w * p.rows * 32 + i].y;
    }
    store_pair(static_cast<T*>(p.query) + (size_t(r) * p.heads + head) * p.row_pad + column, sum.x, sum.y);
  }
}

__device__ __forceinline__ float4 quad_of(const float* p) { return *reinterpret_cast<const float4*>(p); }

// ---- split attention over the cache rows --------------------------------------------------------------------------
constexpr int kTile = 64;
constexpr int kWeightPitch = kTile + 8;  // BF16 elements per staged row of softmax weights

struct LatentShared {
  uint64_t full[2];
  int failed;
  float tops[8][16];
  float sums[8][16];
};

// Byte offset of (token, 16-byte piece of the row) in a tile staged as [64-value piece][token][128 B], 128-byte swizzle.
__device__ __forceinline__ int staged_offset(int token, int piece) {
  const int at = (piece >> 3) * (kTile * 128) + token * 128 + ((piece & 7) << 4);
  return at ^ (((at >> 7) & 7) << 4);
}

size_t latent_shared_bytes(int row_pad, int stages) {
  return size_t(stages) * kTile * row_pad * 2 + size_t(16) * (row_pad + 8) * 2 + size_t(2) * 16 * kWeightPitch * 2 +
         sizeof(LatentShared) + 1024;
}

// Block (split of the sequence, 16 (row, head) pairs). Eight warps share the tile: each scores eight tokens for all 16
// pairs, then sums every eighth 16-value column of the latents, kColumns at most.
constexpr int kWarps = 8;
template <int kColumns>
__global__ void __launch_bounds__(kWarps * 32) latent_attention_kernel(const __grid_constant__ SizedAttentionParams p, int row_pad,
                                                                       int stages) {
  extern __shared__ unsigned char latent_smem_raw[];
  unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(latent_smem_raw) + 1023) & ~uintptr_t(1023));
  const int stage_bytes = kTile * row_pad * 2, query_pitch = row_pad + 8;
  bf16* query = reinterpret_cast<bf16*>(smem + size_t(stages) * stage_bytes);  // [16][row_pad + 8]
  bf16* leading = query + 16 * query_pitch;                                     // [16][kWeightPitch]
  bf16* rest = leading + 16 * kWeightPitch;
  LatentShared* sh = reinterpret_cast<LatentShared*>(rest + 16 * kWeightPitch);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
  const int matrix = lane >> 3, in_matrix = lane & 7;

  const int offset = *p.device_offset;  // written by the previous step
  if (offset < 0 || offset + p.rows > p.capacity) {
    grid_dependency_wait();
    return;
  }
  const int stacked = p.rows * p.heads, first_pair = blockIdx.y * 16;
  const int last_row = min(stacked - 1, first_pair + 15) / p.heads;
  const int split = blockIdx.x, start = split * p.chunk;
  if (start >= offset + p.rows) return;  // beyond every row: no other block's work depends on this one
  const int end = min(start + p.chunk, offset + last_row + 1);
  const int tiles = max(0, (end - start + kTile - 1) / kTile);
  const uint32_t wait_limit = p.wait_limit ? p.wait_limit : kTmaWaitLimit;
  if (threadIdx.x == 0) {
    for (int s = 0; s < stages; ++s) mbarrier_init(&sh->full[s], 1);
    sh->failed = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  __syncthreads();
  auto request = [&](int tile) {
    const int stage = tile % stages;
    mbarrier_expect_tx(&sh->full[stage], uint32_t(stage_bytes) + (tile == 0 ? p.fault_tx : 0u));
    tma_load_3d(smem + size_t(stage) * stage_bytes, &p.k_map, 0, start + tile * kTile, 0, &sh->full[stage]);
  };
  const bool settled = end <= offset;  // nothing in this split is written by the preceding kernel
  if (!settled) grid_dependency_wait();
  if (threadIdx.x == 0)
    for (int tile = 0; tile < min(stages, tiles); ++tile) request(tile);
  if (settled) grid_dependency_wait();
  grid_launch_dependents();

  const int pieces = row_pad / 8;
  for (int i = threadIdx.x; i < 16 * pieces; i += kWarps * 32) {
    const int pair = i / pieces, piece = i - pair * pieces;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (first_pair + pair < stacked)
      v = *reinterpret_cast<const uint4*>(static_cast<const bf16*>(p.q) + size_t(first_pair + pair) * row_pad + piece * 8);
    *reinterpret_cast<uint4*>(query + pair * query_pitch + piece * 8) = v;
  }
  __syncthreads();
  const int limit_lo = first_pair + g < stacked ? offset + (first_pair + g) / p.heads : -1;  // last visible token
  const int limit_hi = first_pair + g + 8 < stacked ? offset + (first_pair + g + 8) / p.heads : -1;
  float o[kColumns][2][4];
#pragma unroll
  for (int j = 0; j < kColumns; ++j)
#pragma unroll
    for (int h = 0; h < 2; ++h) o[j][h][0] = o[j][h][1] = o[j][h][2] = o[j][h][3] = 0.0f;
  float m_lo = -INFINITY, m_hi = -INFINITY, l_lo = 0.0f, l_hi = 0.0f;  // l: this warp's tokens only
  const int columns = p.vdim_pad / 16, steps = row_pad / 16;

  int tile = 0;
  bool gave_up = false;
  for (; tile < tiles; ++tile) {
    const int stage = tile % stages;
    if (!mbarrier_wait(&sh->full[stage], (tile / stages) & 1, wait_limit)) sh->failed = 1;
    unsigned char* rows = smem + size_t(stage) * stage_bytes;
    const int first = start + tile * kTile;
    if (end - first < kTile) {
      // Cache rows beyond the block's history hold whatever was there; their scores are masked and they are cleared, so
      // that a non-finite leftover cannot pass through a zero weight.
      const int live = end - first;
      for (int i = threadIdx.x; i < (kTile - live) * pieces; i += kWarps * 32)
        *reinterpret_cast<uint4*>(rows + staged_offset(live + i / pieces, i % pieces)) = make_uint4(0, 0, 0, 0);
      __syncthreads();
    }
    float s[4], other[4];  // even and odd k-steps: two chains
    s[0] = s[1] = s[2] = s[3] = other[0] = other[1] = other[2] = other[3] = 0.0f;
#pragma unroll 4
    for (int kk = 0; kk < steps; kk += 2) {  // a row has an even number of k-steps
      uint32_t a0, a1, a2, a3, b0, b1, b2, b3;
      ldmatrix_x4(b0, b1, b2, b3, rows + staged_offset(warp * 8 + in_matrix, 2 * kk + matrix));
      ldmatrix_x4(a0, a1, a2, a3, query + ((matrix & 1) * 8 + in_matrix) * query_pitch + kk * 16 + (matrix >> 1) * 8);
      mma_bf16_16816(s, a0, a1, a2, a3, b0, b1);
      ldmatrix_x4(a0, a1, a2, a3, query + ((matrix & 1) * 8 + in_matrix) * query_pitch + (kk + 1) * 16 + (matrix >> 1) * 8);
      mma_bf16_16816(other, a0, a1, a2, a3, b2, b3);
    }
    float top_lo, top_hi;
    const int t0 = first + warp * 8 + 2 * c, t1 = t0 + 1;
    s[0] = t0 <= limit_lo ? (s[0] + other[0]) * p.scale : -INFINITY;
    s[1] = t1 <= limit_lo ? (s[1] + other[1]) * p.scale : -INFINITY;
    s[2] = t0 <= limit_hi ? (s[2] + other[2]) * p.scale : -INFINITY;
    s[3] = t1 <= limit_hi ? (s[3] + other[3]) * p.scale : -INFINITY;
    top_lo = fmaxf(s[0], s[1]);
    top_hi = fmaxf(s[2], s[3]);
#pragma unroll
    for (int d = 1; d <= 2; d <<= 1) {
      top_lo = fmaxf(top_lo, __shfl_xor_sync(0xffffffffu, top_lo, d));
      top_hi = fmaxf(top_hi, __shfl_xor_sync(0xffffffffu, top_hi, d));
    }
    if (c == 0) {
      sh->tops[warp][g] = top_lo;
      sh->tops[warp][g + 8] = top_hi;
    }
    __syncthreads();
    float new_lo = m_lo, new_hi = m_hi;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
      new_lo = fmaxf(new_lo, sh->tops[w][g]);
      new_hi = fmaxf(new_hi, sh->tops[w][g + 8]);
    }
    const float base_lo = new_lo == -INFINITY ? 0.0f : new_lo, base_hi = new_hi == -INFINITY ? 0.0f : new_hi;
    const float rescale_lo = __expf(m_lo - base_lo), rescale_hi = __expf(m_hi - base_hi);
    m_lo = new_lo;
    m_hi = new_hi;
    const float p0 = __expf(s[0] - base_lo), p1 = __expf(s[1] - base_lo);
    const float p2 = __expf(s[2] - base_hi), p3 = __expf(s[3] - base_hi);
    {
      const int at = warp * 8 + 2 * c;
      uint32_t hi, lo;
      split_pair(p0, p1, hi, lo);
      *reinterpret_cast<uint32_t*>(leading + g * kWeightPitch + at) = hi;
      *reinterpret_cast<uint32_t*>(rest + g * kWeightPitch + at) = lo;
      split_pair(p2, p3, hi, lo);
      *reinterpret_cast<uint32_t*>(leading + (g + 8) * kWeightPitch + at) = hi;
      *reinterpret_cast<uint32_t*>(rest + (g + 8) * kWeightPitch + at) = lo;
    }
    l_lo = l_lo * rescale_lo + (p0 + p1);
    l_hi = l_hi * rescale_hi + (p2 + p3);
#pragma unroll
    for (int j = 0; j < kColumns; ++j)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        o[j][h][0] *= rescale_lo;
        o[j][h][1] *= rescale_lo;
        o[j][h][2] *= rescale_hi;
        o[j][h][3] *= rescale_hi;
      }
    __syncthreads();
#pragma unroll
    for (int t = 0; t < kTile / 16; ++t) {
      uint32_t a0, a1, a2, a3, r0, r1, r2, r3;
      const int at = ((matrix & 1) * 8 + in_matrix) * kWeightPitch + t * 16 + (matrix >> 1) * 8;
      ldmatrix_x4(a0, a1, a2, a3, leading + at);
      ldmatrix_x4(r0, r1, r2, r3, rest + at);
#pragma unroll
      for (int j = 0; j < kColumns; ++j) {
        const int column = warp + j * kWarps;
        if (column < columns) {
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4_trans(b0, b1, b2, b3, rows + staged_offset(t * 16 + (matrix & 1) * 8 + in_matrix, 2 * column + (matrix >> 1)));
          mma_bf16_16816(o[j][0], a0, a1, a2, a3, b0, b1);
          mma_bf16_16816(o[j][1], a0, a1, a2, a3, b2, b3);
          mma_bf16_16816(o[j][0], r0, r1, r2, r3, b0, b1);
          mma_bf16_16816(o[j][1], r0, r1, r2, r3, b2, b3);
        }
      }
    }
    __syncthreads();  // every warp is done with this stage, the maxima and the weights
    gave_up = sh->failed != 0;
    if (gave_up) break;
    if (threadIdx.x == 0 && tile + stages < tiles) request(tile + stages);
  }
  if (gave_up) {
    if (threadIdx.x == 0) {
      for (int t = max(tile, p.fault_tx ? 1 : 0); t < min(tile + stages, tiles); ++t)
        mbarrier_wait(&sh->full[t % stages], (t / stages) & 1, wait_limit);
      if (p.status) atomicOr(p.status, 4);
    }
    return;
  }
#pragma unroll
  for (int d = 1; d <= 2; d <<= 1) {
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, d);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, d);
  }
  if (c == 0) {
    sh->sums[warp][g] = l_lo;
    sh->sums[warp][g + 8] = l_hi;
  }
  __syncthreads();
  const int pitch = p.vdim_pad + 4;
  float* to_lo = p.scratch + (size_t(split) * stacked + first_pair + g) * pitch;
  float* to_hi = to_lo + size_t(8) * pitch;
  const bool live_lo = first_pair + g < stacked, live_hi = first_pair + g + 8 < stacked;
#pragma unroll
  for (int j = 0; j < kColumns; ++j) {
    const int column = warp + j * kWarps;
    if (column >= columns) continue;
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int at = column * 16 + h * 8 + 2 * c;
      if (live_lo) *reinterpret_cast<float2*>(to_lo + at) = make_float2(o[j][h][0], o[j][h][1]);
      if (live_hi) *reinterpret_cast<float2*>(to_hi + at) = make_float2(o[j][h][2], o[j][h][3]);
    }
  }
  if (warp == 0 && c == 0) {
    float sum_lo = 0.0f, sum_hi = 0.0f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
      sum_lo += sh->sums[w][g];
      sum_hi += sh->sums[w][g + 8];
    }
    if (live_lo) *reinterpret_cast<float2*>(to_lo + p.vdim_pad) = make_float2(m_lo, sum_lo);
    if (live_hi) *reinterpret_cast<float2*>(to_hi + p.vdim_pad) = make_float2(m_hi, sum_hi);
  }
}

// Block ((row, head), 32 values): the splits are merged into one latent - a thread sums four columns of every second
// split -, every warp then expands four values of it, and the output gate is applied. The expansion's rows are requested
// before waiting for the attention.
constexpr int kExpandThreads = 256;
constexpr int kExpandQuads = 4;   // quads of a row a lane requests ahead: 512 latent values
constexpr int kMergeAhead = 8;    // splits a thread requests at once
template <typename T>
__global__ void __launch_bounds__(kExpandThreads) latent_expand_kernel(const LatentParams p, const SizedAttentionParams a, int merge) {
  __shared__ __align__(16) float latent[kMaxLatent];
  __shared__ __align__(16) float other[kMaxLatent];
  __shared__ float weights[64];
  __shared__ float shared[1];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int offset = *a.device_offset;  // written by the previous step
  const int pair = blockIdx.x, row = pair / p.heads, head = pair - row * p.heads;
  const int first_value = blockIdx.y * 32 + warp * 4;
  const bf16* values = p.expand + (size_t(p.heads) * p.dim_pad + size_t(head) * p.vdim_pad + first_value) * p.rank_pad;
  uint2 held[4][kExpandQuads];
#pragma unroll
  for (int j = 0; j < 4; ++j)
#pragma unroll
    for (int i = 0; i < kExpandQuads; ++i) {
      const int at = (lane + 32 * i) * 4;
      held[j][i] = make_uint2(0, 0);
      if (first_value + j < p.vdim_pad && at < p.rank_pad) held[j][i] = *reinterpret_cast<const uint2*>(values + size_t(j) * p.rank_pad + at);
    }
  grid_dependency_wait();
  grid_launch_dependents();
  if (offset < 0 || offset + p.rows > p.capacity) return;
  if (merge) {
    const int splits = min(64, (offset + p.rows + a.chunk - 1) / a.chunk), pitch = p.rank_pad + 4;
    const float* base = a.scratch + size_t(pair) * pitch;
    const size_t step = size_t(p.rows) * p.heads * pitch;
    const int half = threadIdx.x >> 7, column = (threadIdx.x & 127) * 4;  // splits half, half + 2, ..
    float4 x[kMergeAhead];
    auto request = [&](int s, int at) {
#pragma unroll
      for (int i = 0; i < kMergeAhead; ++i) {
        x[i] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (s + 2 * i < splits && at < p.rank_pad) x[i] = quad_of(base + (s + 2 * i) * step + at);
      }
    };
    request(half, column);
    if (warp == 0) {
      float m[2], l[2];
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int s = lane + 32 * h;
        const float2 ml = s < splits ? *reinterpret_cast<const float2*>(base + s * step + p.rank_pad) : make_float2(-INFINITY, 0.0f);
        m[h] = ml.x;
        l[h] = ml.y;
      }
      const float top = warp_max(fmaxf(m[0], m[1]));
      float sum = 0.0f;
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const float w = m[h] == -INFINITY ? 0.0f : expf(m[h] - top);
        weights[lane + 32 * h] = w;
        sum += w * l[h];
      }
      sum = warp_sum(sum);
      if (lane == 0) shared[0] = sum > 0.0f ? 1.0f / sum : 0.0f;
    }
    __syncthreads();
    for (int at = column; at < p.rank_pad; at += 512) {
      float4 sum = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
      for (int s = half; s < splits; s += 2 * kMergeAhead) {
        if (s != half || at != column) request(s, at);
        // A split in which this pair saw nothing has weight zero and finite sums.
#pragma unroll
        for (int i = 0; i < kMergeAhead; ++i) {
          const float w = s + 2 * i < splits ? weights[s + 2 * i] : 0.0f;
          sum = make_float4(fmaf(w, x[i].x, sum.x), fmaf(w, x[i].y, sum.y), fmaf(w, x[i].z, sum.z), fmaf(w, x[i].w, sum.w));
        }
      }
      *reinterpret_cast<float4*>((half ? other : latent) + at) = sum;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < p.rank_pad; i += kExpandThreads) latent[i] = (latent[i] + other[i]) * shared[0];
  } else {
    const T* from = static_cast<const T*>(a.out) + size_t(row) * a.out_stride + size_t(head) * p.rank_pad;
    for (int i = threadIdx.x; i < p.rank_pad; i += kExpandThreads) latent[i] = value_of(from[i]);
  }
  __syncthreads();
  const T* gate = static_cast<const T*>(p.fused) + size_t(row) * p.stride + p.gate_at + size_t(head) * p.vdim_pad;
  T* out = static_cast<T*>(p.out) + size_t(row) * p.out_stride + size_t(head) * p.vdim_pad;
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int v = first_value + j;
    if (v >= p.vdim_pad) break;
    float sum = 0.0f;
    auto add_quad = [&](int at, float4 w) {
      const float4 y = quad_of(latent + at);
      sum = fmaf(w.x, y.x, fmaf(w.y, y.y, fmaf(w.z, y.z, fmaf(w.w, y.w, sum))));
    };
#pragma unroll
    for (int i = 0; i < kExpandQuads; ++i) {
      const int at = (lane + 32 * i) * 4;
      if (at < p.rank_pad)
        add_quad(at, make_float4(bf16_lo(held[j][i].x), bf16_hi(held[j][i].x), bf16_lo(held[j][i].y), bf16_hi(held[j][i].y)));
    }
    for (int at = (lane + 32 * kExpandQuads) * 4; at < p.rank_pad; at += 128) add_quad(at, load_quad(values + size_t(j) * p.rank_pad + at));
    sum = warp_sum(sum);
    if (lane == 0) store_value(out + v, sum * sigmoid_for<T>(value_of(gate[v])));
  }
  if (head == 0 && blockIdx.y == 0) {
    T* end = static_cast<T*>(p.out) + size_t(row) * p.out_stride;
    for (int i = p.heads * p.vdim_pad + threadIdx.x; i < p.out_stride; i += kExpandThreads) store_value(end + i, 0.0f);
  }
}

int latent_stages(int row_pad, size_t smem_limit) { return latent_shared_bytes(row_pad, 2) <= smem_limit ? 2 : 1; }

template <int kColumns>
void launch_latent_columns(const SizedAttentionParams& p, int row_pad, size_t smem_limit, cudaStream_t stream, bool pdl) {
  static thread_local int configured_device = -1;
  int device = 0;
  EI_CUDA(cudaGetDevice(&device));
  if (configured_device != device) {
    EI_CUDA(cudaFuncSetAttribute(latent_attention_kernel<kColumns>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem_limit) - 1024));
    configured_device = device;
  }
  const int stages = latent_stages(row_pad, smem_limit - 1024);
  launch(latent_attention_kernel<kColumns>, dim3(unsigned(p.max_splits), unsigned((p.rows * p.heads + 15) / 16)), dim3(kWarps * 32),
         latent_shared_bytes(row_pad, stages), stream, pdl, p, row_pad, stages);
}

}  // namespace

namespace {
template <typename T, int kRows>
void launch_prepare_rows(const LatentParams& p, bool step, cudaStream_t stream, bool pdl) {
  static thread_local int configured_device = -1;
  int device = 0;
  EI_CUDA(cudaGetDevice(&device));
  if (configured_device != device) {
    EI_CUDA(cudaFuncSetAttribute(latent_prepare_kernel<T, kRows>, cudaFuncAttributeMaxDynamicSharedMemorySize, kRows * (kMaxHeadDim * 4 + 2048)));
    configured_device = device;
  }
  const int absorbing = step ? p.heads * (p.rank_pad / 64) : 0;
  const size_t smem = step ? size_t(p.rows) * (p.dim_pad * 4 + 2048) : 0;
  const int quads = (step ? p.row_pad - p.rank_pad : p.rot_pad) / 4;
  const int blocks = absorbing + (p.rows + 7) / 8 + (p.rows * p.heads * quads + kPrepareThreads - 1) / kPrepareThreads;
  launch(latent_prepare_kernel<T, kRows>, dim3(unsigned(blocks)), dim3(kPrepareThreads), smem, stream, pdl, p, absorbing);
}
}  // namespace

template <typename T>
void launch_latent_prepare(const LatentParams& p, bool step, cudaStream_t stream, bool pdl) {
  if (step && (p.rows > kMaxRows || p.dim_pad > kMaxHeadDim)) throw std::invalid_argument("a latent attention step takes 1..16 rows");
  if (!step || p.rows == 1) return launch_prepare_rows<T, 1>(p, step, stream, pdl);
  if (p.rows <= 4) return launch_prepare_rows<T, 4>(p, step, stream, pdl);
  launch_prepare_rows<T, kMaxRows>(p, step, stream, pdl);
}

bool latent_attention_ok(int rank_pad, int row_pad, size_t smem_limit) {
  return rank_pad <= kMaxLatent && latent_shared_bytes(row_pad, 1) <= smem_limit - 1024;
}

void launch_latent_attention(const SizedAttentionParams& given, int row_pad, size_t smem_limit, cudaStream_t stream, bool pdl) {
  SizedAttentionParams p = given;
  if (!latent_attention_ok(p.vdim_pad, row_pad, smem_limit)) throw std::invalid_argument("latent beyond the tiled attention's range");
  const cuuint64_t dims[3] = {64, cuuint64_t((p.capacity + kTile - 1) / kTile * kTile), cuuint64_t(row_pad / 64)};
  const cuuint64_t strides[2] = {cuuint64_t(row_pad) * 2, 128};
  const cuuint32_t box[3] = {64, kTile, cuuint32_t(row_pad / 64)};
  encode_map(&p.k_map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, p.k, dims, strides, box, CU_TENSOR_MAP_SWIZZLE_128B, "latent cache");
  if (p.vdim_pad <= 512)
    launch_latent_columns<4>(p, row_pad, smem_limit, stream, pdl);
  else
    launch_latent_columns<8>(p, row_pad, smem_limit, stream, pdl);
}

template <typename T>
void launch_latent_expand(const LatentParams& p, const SizedAttentionParams& a, bool merge, cudaStream_t stream, bool pdl) {
  launch(latent_expand_kernel<T>, dim3(unsigned(p.rows * p.heads), unsigned((p.vdim_pad + 31) / 32)), dim3(kExpandThreads), 0,
         stream, pdl, p, a, merge ? 1 : 0);
}

template void launch_latent_prepare<bf16>(const LatentParams&, bool, cudaStream_t, bool);
template void launch_latent_prepare<float>(const LatentParams&, bool, cudaStream_t, bool);
template void launch_latent_expand<bf16>(const LatentParams&, const SizedAttentionParams&, bool, cudaStream_t, bool);
template void launch_latent_expand<float>(const LatentParams&, const SizedAttentionParams&, bool, cudaStream_t, bool);

}  // namespace ei
