// Decayed linear attention. Per head a matrix M (key size x value size, FP32) becomes decay M + k v^T with every row,
// and the row's output is q^T M.
//
// A step of at most 16 rows leaves its rows pending: their k and v stay in a ring indexed by position and the next
// step folds those that were kept into the state it reads anyway, so a rejected draft costs nothing and no copy of a
// state is ever taken. The state holds the first Control::state_base rows; rows [state_base, context) are pending.
//
// A prompt segment runs in chunks of 128 tokens, three launches whose work is parallel over chunks, heads and value
// slices: the chunks' own contributions sum_j decay^(n-1-j) k_j v_j^T; a scan over chunks that turns them into the
// state ahead of every chunk (and the final state); and the outputs, decay^(i+1) q_i S + sum_(j<=i) decay^(i-j)
// (q_i . k_j) v_j. The matrix products run on mma.sync with FP32 sums; what is FP32 by nature (the state, the decayed
// values, the decayed scores) enters as two BF16 terms, i.e. with 16 significant bits.
//
// State layout: [head][slice of 16 values][key dimension][16], so that a block streams contiguous memory.
//
// The prompt kernels also run a state-space layer, whose decay and write strength belong to the token (TokenDecay): the
// powers of the head's decay become exponentials of differences of cumulative logarithms, never above zero. Its step form
// is in outer_state.cu.
#include "layered_device.cuh"

#include <stdexcept>

namespace ei {
namespace {

constexpr int kStepThreads = 128;
constexpr int kDimStep = kStepThreads / 4;       // key dimensions a block covers at once: 4 threads x float4 = 16 values
constexpr int kStrips = 8;                       // strips held in registers: 256 key dimensions

size_t step_shared_floats(int rows_bucket, int dim_pad) {
  return size_t(2 * rows_bucket + kPendingRows) * dim_pad     // q and k of the step, k of the pending rows
         + size_t(kPendingRows + rows_bucket) * 16             // values of the slice
         + size_t((rows_bucket * rows_bucket + 3) & ~3)        // decayed scores inside the step
         + size_t(4) * rows_bucket * 16;                       // the warps' partial outputs
}

template <typename T, int kRows>
__global__ void __launch_bounds__(kStepThreads) lightning_step_kernel(const LightningParams p) {
  extern __shared__ float step_smem[];
  float* q_rows = step_smem;                                   // [kRows][dim]
  float* k_rows = q_rows + size_t(kRows) * p.dim_pad;          // [kPendingRows + kRows][dim]
  float* v_rows = k_rows + size_t(kPendingRows + kRows) * p.dim_pad;  // [kPendingRows + kRows][16]
  float* scores = v_rows + (kPendingRows + kRows) * 16;        // [kRows][kRows]
  float* parts = scores + ((kRows * kRows + 3) & ~3);          // [4][kRows][16]
  const int head = blockIdx.x, slice = blockIdx.y, dim = p.dim_pad;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // Written by the previous step, several kernels ago: read, and the state requested, before waiting.
  const int context = p.control->context, base = p.control->state_base;
  const bool runs = context >= 0 && context + p.rows <= p.capacity;
  const int pending = min(kPendingRows, max(0, context - base));
  float* state = p.state + (size_t(head) * (p.vdim_pad / 16) + slice) * dim * 16 + (threadIdx.x & 3) * 4;
  const int d0 = threadIdx.x >> 2;
  float4 held[kStrips];
#pragma unroll
  for (int i = 0; i < kStrips; ++i) {
    const int d = d0 + i * kDimStep;
    held[i] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (runs && base > 0 && d < dim) held[i] = *reinterpret_cast<const float4*>(state + size_t(d) * 16);
  }
  const float* powers = p.powers + size_t(head) * (kLightningChunk + 1);
  grid_dependency_wait();
  grid_launch_dependents();
  if (!runs) return;

  const T* ring_k = static_cast<const T*>(p.ring_k);
  const T* ring_v = static_cast<const T*>(p.ring_v);
  const size_t k_pitch = size_t(p.heads) * dim, v_pitch = size_t(p.heads) * p.vdim_pad;
  const int known = pending + p.rows;
  for (int i = threadIdx.x; i < known * dim; i += kStepThreads) {
    const int row = i / dim, d = i - row * dim;
    k_rows[i] = value_of(ring_k[size_t((base + row) & (kRingRows - 1)) * k_pitch + size_t(head) * dim + d]);
  }
  for (int i = threadIdx.x; i < p.rows * dim; i += kStepThreads) {
    const int row = i / dim, d = i - row * dim;
    q_rows[i] = value_of(static_cast<const T*>(p.q)[size_t(row) * p.stride + size_t(head) * dim + d]);
  }
  for (int i = threadIdx.x; i < known * 16; i += kStepThreads)
    v_rows[i] = value_of(ring_v[size_t((base + (i >> 4)) & (kRingRows - 1)) * v_pitch + size_t(head) * p.vdim_pad +
                                slice * 16 + (i & 15)]);
  __syncthreads();

  // Decayed scores of the step's own rows: a warp per (row, earlier row).
  for (int pair = warp; pair < p.rows * p.rows; pair += kStepThreads / 32) {
    const int r = pair / p.rows, j = pair - r * p.rows;
    if (j > r) continue;
    float sum = 0.0f;
    for (int d = lane; d < dim; d += 32) sum = fmaf(q_rows[r * dim + d], k_rows[(pending + j) * dim + d], sum);
    sum = warp_sum(sum);
    if (lane == 0) scores[r * kRows + j] = sum * powers[r - j];
  }

  float4 acc[kRows];
#pragma unroll
  for (int r = 0; r < kRows; ++r) acc[r] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  const float whole = powers[pending];
  const int column = (threadIdx.x & 3) * 4;
  for (int first = 0; first < dim; first += kStrips * kDimStep) {
#pragma unroll
    for (int i = 0; i < kStrips; ++i) {
      const int d = first + d0 + i * kDimStep;
      if (d >= dim) continue;
      float4 s = held[i];
      if (first > 0) s = base > 0 ? *reinterpret_cast<const float4*>(state + size_t(d) * 16) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
      if (pending) {
        s.x *= whole; s.y *= whole; s.z *= whole; s.w *= whole;
        for (int j = 0; j < pending; ++j) {
          const float k = k_rows[j * dim + d] * powers[pending - 1 - j];
          const float4 v = *reinterpret_cast<const float4*>(v_rows + j * 16 + column);
          s.x = fmaf(k, v.x, s.x); s.y = fmaf(k, v.y, s.y); s.z = fmaf(k, v.z, s.z); s.w = fmaf(k, v.w, s.w);
        }
        *reinterpret_cast<float4*>(state + size_t(d) * 16) = s;
      }
#pragma unroll
      for (int r = 0; r < kRows; ++r) {
        if (r < p.rows) {
          const float q = q_rows[r * dim + d];
          acc[r].x = fmaf(q, s.x, acc[r].x); acc[r].y = fmaf(q, s.y, acc[r].y);
          acc[r].z = fmaf(q, s.z, acc[r].z); acc[r].w = fmaf(q, s.w, acc[r].w);
        }
      }
    }
  }
  // Sum over the key dimensions: the eight lanes of a column group, then the four warps.
#pragma unroll
  for (int r = 0; r < kRows; ++r) {
#pragma unroll
    for (int o = 4; o <= 16; o <<= 1) {
      acc[r].x += __shfl_xor_sync(0xffffffffu, acc[r].x, o);
      acc[r].y += __shfl_xor_sync(0xffffffffu, acc[r].y, o);
      acc[r].z += __shfl_xor_sync(0xffffffffu, acc[r].z, o);
      acc[r].w += __shfl_xor_sync(0xffffffffu, acc[r].w, o);
    }
    if (lane < 4) *reinterpret_cast<float4*>(parts + (warp * kRows + r) * 16 + lane * 4) = acc[r];
  }
  __syncthreads();
  for (int i = threadIdx.x; i < p.rows * 16; i += kStepThreads) {
    const int r = i >> 4, col = i & 15;
    float inter = 0.0f;
#pragma unroll
    for (int w = 0; w < 4; ++w) inter += parts[(w * kRows + r) * 16 + col];
    float sum = inter * powers[r + 1];
    for (int j = 0; j <= r; ++j) sum = fmaf(scores[r * kRows + j], v_rows[(pending + j) * 16 + col], sum);
    p.out[size_t(r) * v_pitch + size_t(head) * p.vdim_pad + slice * 16 + col] = sum;
  }
}

// ---- prompt segments ------------------------------------------------------------------------------------------
constexpr int kChunk = kLightningChunk;
constexpr int kSlice = 64;               // values per block
constexpr int kPitch = kSlice + 8;       // BF16 elements per staged value row: an odd number of 16-byte pieces
constexpr int kPromptThreads = 256;

// Requests a 16-byte piece into shared memory; a dead piece is filled with zeros and not read.
__device__ __forceinline__ void request_piece(bf16* to, const bf16* from, bool live) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_address(to)), "l"(from), "r"(live ? 16 : 0) : "memory");
}
__device__ __forceinline__ void await_pieces() { asm volatile("cp.async.wait_all;" ::: "memory"); }
// Requests rows [0, live) of a [tokens][dim] BF16 operand, zeros behind them.
__device__ __forceinline__ void stage_rows(bf16* to, const bf16* from, int stride, int live, int pieces, int pitch) {
#pragma unroll 8
  for (int i = threadIdx.x; i < kChunk * pieces; i += kPromptThreads) {
    const int row = i / pieces, piece = i - row * pieces;
    request_piece(to + size_t(row) * pitch + piece * 8, from + (row < live ? size_t(row) * stride : 0) + piece * 8, row < live);
  }
}

// Logarithms of the decays from the chunk's start through each of its rows, and the rows' steps; `cumulative` [kChunk]
// and `strengths` [kChunk] are complete after the next block-wide barrier. All threads of the block take part.
__device__ __forceinline__ void token_decays(const TokenDecay& t, int head, int first, int live, float* cumulative,
                                             float* strengths, float* warp_totals) {
  static_assert(kChunk == 128, "four warps scan a chunk");
  const int row = threadIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float sum = 0.0f;
  if (row < kChunk) {
    float step = 0.0f;
    if (row < live) step = softplus_value(__bfloat162float(t.step[size_t(first + row) * t.step_stride + head]) + t.bias[head]);
    strengths[row] = step;
    sum = -t.rate[head] * step;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float below = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += below;
    }
    if (lane == 31) warp_totals[warp] = sum;
  }
  __syncthreads();
  if (row < kChunk) {
    for (int w = 0; w < warp; ++w) sum += warp_totals[w];
    cumulative[row] = sum;
  }
}

size_t chunk_state_shared(int dim_pad) { return size_t(kChunk) * (dim_pad + 8) * 2 + size_t(2) * kChunk * kPitch * 2; }

// Block (chunk, head, slice of 64 values): chunk_states[chunk][head] = sum_j decay^(n-1-j) k_j v_j^T.
template <bool kToken>
__global__ void __launch_bounds__(kPromptThreads) lightning_chunk_kernel(const LightningParams p) {
  extern __shared__ __align__(16) unsigned char chunk_smem[];
  const int dim = p.dim_pad, k_pitch = dim + 8;
  bf16* keys = reinterpret_cast<bf16*>(chunk_smem);            // [kChunk][dim + 8]
  bf16* leading = keys + size_t(kChunk) * k_pitch;             // [kChunk][kPitch]
  bf16* rest = leading + kChunk * kPitch;
  grid_dependency_wait();
  grid_launch_dependents();
  const int context = p.control->context;
  if (context < 0 || context + p.rows > p.capacity) return;
  const int chunk = blockIdx.x, head = blockIdx.y, first_value = blockIdx.z * kSlice;
  const int first = chunk * kChunk, live = min(kChunk, p.rows - first);
  const int values = min(kSlice, p.vdim_pad - first_value);
  const float* powers = kToken ? nullptr : p.powers + size_t(head) * (kChunk + 1);
  const int key_head = kToken ? head / (p.heads / p.token.key_heads) : head;
  stage_rows(keys, static_cast<const bf16*>(p.k) + size_t(first) * p.stride + size_t(key_head) * dim, p.stride, live, dim / 8,
             k_pitch);
  __shared__ float cumulative[kToken ? kChunk : 1], strengths[kToken ? kChunk : 1], warp_totals[4];
  if (kToken) {
    token_decays(p.token, head, first, live, cumulative, strengths, warp_totals);
    __syncthreads();
    if (threadIdx.x == 0 && blockIdx.z == 0) p.token.totals[size_t(chunk) * p.heads + head] = cumulative[kChunk - 1];
  }
#pragma unroll
  for (int i = threadIdx.x; i < kChunk * (kSlice / 8); i += kPromptThreads) {
    const int row = i >> 3, piece = i & 7;
    uint4 hi = make_uint4(0, 0, 0, 0), lo = hi;
    if (row < live && piece * 8 < values) {
      const uint4 v = *reinterpret_cast<const uint4*>(static_cast<const bf16*>(p.v) + size_t(first + row) * p.stride +
                                                      size_t(head) * p.vdim_pad + first_value + piece * 8);
      const float w = kToken ? __expf(cumulative[kChunk - 1] - cumulative[row]) * strengths[row] : powers[live - 1 - row];
      split_pair(bf16_lo(v.x) * w, bf16_hi(v.x) * w, hi.x, lo.x);
      split_pair(bf16_lo(v.y) * w, bf16_hi(v.y) * w, hi.y, lo.y);
      split_pair(bf16_lo(v.z) * w, bf16_hi(v.z) * w, hi.z, lo.z);
      split_pair(bf16_lo(v.w) * w, bf16_hi(v.w) * w, hi.w, lo.w);
    }
    *reinterpret_cast<uint4*>(leading + row * kPitch + piece * 8) = hi;
    *reinterpret_cast<uint4*>(rest + row * kPitch + piece * 8) = lo;
  }
  await_pieces();
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
  const int matrix = lane >> 3, in_matrix = lane & 7;
  const int steps = (live + 15) / 16;
  for (int tile = warp; tile < dim / 16; tile += kPromptThreads / 32) {
    float acc[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.0f;
    for (int t = 0; t < steps; ++t) {
      uint32_t a0, a1, a2, a3;  // rows = key dimensions, columns = tokens: the transpose of the staged keys
      ldmatrix_x4_trans(a0, a1, a2, a3, keys + size_t(t * 16 + (matrix >> 1) * 8 + in_matrix) * k_pitch + tile * 16 + (matrix & 1) * 8);
#pragma unroll
      for (int n = 0; n < 8; n += 2) {
        const int at = (t * 16 + (matrix & 1) * 8 + in_matrix) * kPitch + (n + (matrix >> 1)) * 8;
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(b0, b1, b2, b3, leading + at);
        mma_bf16_16816(acc[n], a0, a1, a2, a3, b0, b1);
        mma_bf16_16816(acc[n + 1], a0, a1, a2, a3, b2, b3);
        ldmatrix_x4_trans(b0, b1, b2, b3, rest + at);
        mma_bf16_16816(acc[n], a0, a1, a2, a3, b0, b1);
        mma_bf16_16816(acc[n + 1], a0, a1, a2, a3, b2, b3);
      }
    }
    const size_t head_floats = size_t(dim) * p.vdim_pad;
    float* out = p.chunk_states + (size_t(chunk) * p.heads + head) * head_floats;
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      const int value = first_value + n * 8 + 2 * c;
      if (n * 8 >= values) continue;
      float* to = out + (size_t(value >> 4) * dim + tile * 16 + g) * 16 + (value & 15);
      *reinterpret_cast<float2*>(to) = make_float2(acc[n][0], acc[n][1]);
      *reinterpret_cast<float2*>(to + 8 * 16) = make_float2(acc[n][2], acc[n][3]);
    }
  }
}

// A thread owns four values of one key dimension: folds the pending rows into the state, then walks the chunks,
// replacing each contribution by the state ahead of it; the state after the last chunk goes back.
template <bool kToken>
__global__ void __launch_bounds__(256) lightning_scan_kernel(const LightningParams p) {
  grid_dependency_wait();
  grid_launch_dependents();
  const int context = p.control->context, base = p.control->state_base;
  if (context < 0 || context + p.rows > p.capacity) return;
  const int pending = min(kPendingRows, max(0, context - base));
  const int dim = p.dim_pad, slices = p.vdim_pad / 16;
  const size_t quads = size_t(p.heads) * slices * dim * 4;
  const size_t i = size_t(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= quads) return;
  const int column = int(i & 3) * 4;
  const int d = int((i >> 2) % dim), slice = int((i >> 2) / dim % slices), head = int((i >> 2) / dim / slices);
  const float* powers = kToken ? nullptr : p.powers + size_t(head) * (kChunk + 1);
  float4* state = reinterpret_cast<float4*>(p.state) + i;
  float4 s = base > 0 ? *state : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  if (kToken) {
    const int key_head = head / (p.heads / p.token.key_heads);
    for (int j = 0; j < pending; ++j) {
      const size_t slot = (base + j) & (kRingRows - 1);
      const float k = p.token.ring_k[(slot * p.token.key_heads + key_head) * dim + d], g = p.token.ring_g[slot * p.heads + head];
      const float4 u = *reinterpret_cast<const float4*>(p.token.ring_u + (slot * p.heads + head) * p.vdim_pad + slice * 16 + column);
      s = make_float4(fmaf(k, u.x, g * s.x), fmaf(k, u.y, g * s.y), fmaf(k, u.z, g * s.z), fmaf(k, u.w, g * s.w));
    }
  } else if (pending) {
    const float whole = powers[pending];
    s.x *= whole; s.y *= whole; s.z *= whole; s.w *= whole;
    for (int j = 0; j < pending; ++j) {
      const int slot = (base + j) & (kRingRows - 1);
      const float k = value_of(static_cast<const bf16*>(p.ring_k)[(size_t(slot) * p.heads + head) * dim + d]) * powers[pending - 1 - j];
      const uint2 raw = *reinterpret_cast<const uint2*>(static_cast<const bf16*>(p.ring_v) +
                                                        (size_t(slot) * p.heads + head) * p.vdim_pad + slice * 16 + column);
      s.x = fmaf(k, bf16_lo(raw.x), s.x); s.y = fmaf(k, bf16_hi(raw.x), s.y);
      s.z = fmaf(k, bf16_lo(raw.y), s.z); s.w = fmaf(k, bf16_hi(raw.y), s.w);
    }
  }
  const int chunks = (p.rows + kChunk - 1) / kChunk;
  float4* own = reinterpret_cast<float4*>(p.chunk_states) + i;
  float4 next = *own;
  for (int chunk = 0; chunk < chunks; ++chunk) {
    const float4 add = next;
    if (chunk + 1 < chunks) next = own[size_t(chunk + 1) * quads];
    own[size_t(chunk) * quads] = s;
    const float whole = kToken ? expf(p.token.totals[size_t(chunk) * p.heads + head]) : powers[min(kChunk, p.rows - chunk * kChunk)];
    s.x = fmaf(whole, s.x, add.x); s.y = fmaf(whole, s.y, add.y);
    s.z = fmaf(whole, s.z, add.z); s.w = fmaf(whole, s.w, add.w);
  }
  *state = s;
}

size_t output_shared(int dim_pad) {
  return size_t(kChunk) * (dim_pad + 8) * 2 + size_t(kChunk) * kPitch * 2 + size_t(2) * dim_pad * kPitch * 2 +
         (kChunk + 1) * sizeof(float);
}

// Block (chunk, head, slice of 64 values), eight warps of 16 tokens each.
template <bool kToken>
__global__ void __launch_bounds__(kPromptThreads) lightning_output_kernel(const LightningParams p) {
  extern __shared__ __align__(16) unsigned char output_smem[];
  const int dim = p.dim_pad, k_pitch = dim + 8;
  bf16* keys = reinterpret_cast<bf16*>(output_smem);           // [kChunk][dim + 8]
  bf16* vals = keys + size_t(kChunk) * k_pitch;                // [kChunk][kPitch]
  bf16* leading = vals + kChunk * kPitch;                      // state [dim][kPitch], two terms
  bf16* rest = leading + size_t(dim) * kPitch;
  float* powers = reinterpret_cast<float*>(rest + size_t(dim) * kPitch);
  grid_dependency_wait();
  grid_launch_dependents();
  const int context = p.control->context;
  if (context < 0 || context + p.rows > p.capacity) return;
  const int chunk = blockIdx.x, head = blockIdx.y, first_value = blockIdx.z * kSlice;
  const int first = chunk * kChunk, live = min(kChunk, p.rows - first);
  const int values = min(kSlice, p.vdim_pad - first_value);
  __shared__ float cumulative[kToken ? kChunk : 1], strengths[kToken ? kChunk : 1], warp_totals[4];
  if (!kToken)
    for (int i = threadIdx.x; i <= kChunk; i += blockDim.x) powers[i] = p.powers[size_t(head) * (kChunk + 1) + i];
  const int key_head = kToken ? head / (p.heads / p.token.key_heads) : head;
  stage_rows(keys, static_cast<const bf16*>(p.k) + size_t(first) * p.stride + size_t(key_head) * dim, p.stride, live, dim / 8,
             k_pitch);
  if (kToken) token_decays(p.token, head, first, live, cumulative, strengths, warp_totals);
  {
    const bf16* v = static_cast<const bf16*>(p.v) + size_t(first) * p.stride + size_t(head) * p.vdim_pad + first_value;
#pragma unroll
    for (int i = threadIdx.x; i < kChunk * (kSlice / 8); i += kPromptThreads) {
      const int row = i >> 3, piece = i & 7;
      const bool on = row < live && piece * 8 < values;
      request_piece(vals + row * kPitch + piece * 8, on ? v + size_t(row) * p.stride + piece * 8 : v, on);
    }
  }
  const float* state = p.chunk_states + (size_t(chunk) * p.heads + head) * dim * p.vdim_pad;
#pragma unroll 8
  for (int i = threadIdx.x; i < dim * (kSlice / 4); i += kPromptThreads) {
    const int quad = i & 3, d = (i >> 2) % dim, slice = (i >> 2) / dim;  // consecutive threads: one slice's memory order
    const int value = slice * 16 + quad * 4;
    float4 s = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (value < values)
      s = *reinterpret_cast<const float4*>(state + (size_t((first_value + value) >> 4) * dim + d) * 16 + quad * 4);
    uint2 hi, lo;
    split_pair(s.x, s.y, hi.x, lo.x);
    split_pair(s.z, s.w, hi.y, lo.y);
    *reinterpret_cast<uint2*>(leading + size_t(d) * kPitch + value) = hi;
    *reinterpret_cast<uint2*>(rest + size_t(d) * kPitch + value) = lo;
  }
  await_pieces();
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
  const int matrix = lane >> 3, in_matrix = lane & 7;
  const int lo_row = warp * 16 + g, hi_row = lo_row + 8;
  if (warp * 16 >= live) return;
  const bf16* q = static_cast<const bf16*>(p.q) + size_t(first) * p.stride + size_t(key_head) * dim;
  const int key_tiles = 2 * (warp + 1);  // tiles of eight keys this warp's rows can see
  float acc[8][4], s[16][4];
#pragma unroll
  for (int n = 0; n < 8; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.0f;
#pragma unroll
  for (int n = 0; n < 16; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.0f;
  for (int kk = 0; kk < dim / 16; ++kk) {
    uint32_t a0 = 0, a1 = 0, a2 = 0, a3 = 0;
    if (lo_row < live) {
      a0 = *reinterpret_cast<const uint32_t*>(q + size_t(lo_row) * p.stride + kk * 16 + 2 * c);
      a2 = *reinterpret_cast<const uint32_t*>(q + size_t(lo_row) * p.stride + kk * 16 + 8 + 2 * c);
    }
    if (hi_row < live) {
      a1 = *reinterpret_cast<const uint32_t*>(q + size_t(hi_row) * p.stride + kk * 16 + 2 * c);
      a3 = *reinterpret_cast<const uint32_t*>(q + size_t(hi_row) * p.stride + kk * 16 + 8 + 2 * c);
    }
#pragma unroll
    for (int n = 0; n < 8; n += 2) {
      const size_t at = size_t(kk * 16 + (matrix & 1) * 8 + in_matrix) * kPitch + (n + (matrix >> 1)) * 8;
      uint32_t b0, b1, b2, b3;
      ldmatrix_x4_trans(b0, b1, b2, b3, leading + at);
      mma_bf16_16816(acc[n], a0, a1, a2, a3, b0, b1);
      mma_bf16_16816(acc[n + 1], a0, a1, a2, a3, b2, b3);
      ldmatrix_x4_trans(b0, b1, b2, b3, rest + at);
      mma_bf16_16816(acc[n], a0, a1, a2, a3, b0, b1);
      mma_bf16_16816(acc[n + 1], a0, a1, a2, a3, b2, b3);
    }
#pragma unroll
    for (int n = 0; n < 16; n += 2) {
      if (n < key_tiles) {
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4(b0, b1, b2, b3, keys + size_t((n + (matrix >> 1)) * 8 + in_matrix) * k_pitch + kk * 16 + (matrix & 1) * 8);
        mma_bf16_16816(s[n], a0, a1, a2, a3, b0, b1);
        mma_bf16_16816(s[n + 1], a0, a1, a2, a3, b2, b3);
      }
    }
  }
  // What a row's query sees of the state ahead of the chunk, and of the write of row j of the chunk.
  const float lo_power = kToken ? __expf(cumulative[lo_row]) : powers[lo_row + 1];
  const float hi_power = kToken ? __expf(cumulative[hi_row]) : powers[hi_row + 1];
  auto reach = [&](int row, int j) {
    return kToken ? __expf(cumulative[row] - cumulative[j]) * strengths[j] : powers[row - j];
  };
#pragma unroll
  for (int n = 0; n < 8; ++n) {
    acc[n][0] *= lo_power;
    acc[n][1] *= lo_power;
    acc[n][2] *= hi_power;
    acc[n][3] *= hi_power;
  }
#pragma unroll
  for (int t = 0; t < 8; ++t) {
    if (t <= warp) {
      uint32_t wl[4], wr[4];  // decayed scores of 16 rows x 16 keys as an A operand, two terms
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int n = 2 * t + half, j0 = n * 8 + 2 * c, j1 = j0 + 1;
        const float s0 = j0 <= lo_row ? s[n][0] * reach(lo_row, j0) : 0.0f;
        const float s1 = j1 <= lo_row ? s[n][1] * reach(lo_row, j1) : 0.0f;
        const float s2 = j0 <= hi_row ? s[n][2] * reach(hi_row, j0) : 0.0f;
        const float s3 = j1 <= hi_row ? s[n][3] * reach(hi_row, j1) : 0.0f;
        split_pair(s0, s1, wl[2 * half], wr[2 * half]);
        split_pair(s2, s3, wl[2 * half + 1], wr[2 * half + 1]);
      }
#pragma unroll
      for (int n = 0; n < 8; n += 2) {
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(b0, b1, b2, b3, vals + (t * 16 + (matrix & 1) * 8 + in_matrix) * kPitch + (n + (matrix >> 1)) * 8);
        mma_bf16_16816(acc[n], wl[0], wl[1], wl[2], wl[3], b0, b1);
        mma_bf16_16816(acc[n + 1], wl[0], wl[1], wl[2], wl[3], b2, b3);
        mma_bf16_16816(acc[n], wr[0], wr[1], wr[2], wr[3], b0, b1);
        mma_bf16_16816(acc[n + 1], wr[0], wr[1], wr[2], wr[3], b2, b3);
      }
    }
  }
  if (kToken && p.token.skip) {
    const float skip = p.token.skip[head];
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      const uint32_t lo = *reinterpret_cast<const uint32_t*>(vals + lo_row * kPitch + n * 8 + 2 * c);
      const uint32_t hi = *reinterpret_cast<const uint32_t*>(vals + hi_row * kPitch + n * 8 + 2 * c);
      acc[n][0] = fmaf(skip, bf16_lo(lo), acc[n][0]);
      acc[n][1] = fmaf(skip, bf16_hi(lo), acc[n][1]);
      acc[n][2] = fmaf(skip, bf16_lo(hi), acc[n][2]);
      acc[n][3] = fmaf(skip, bf16_hi(hi), acc[n][3]);
    }
  }
  const size_t pitch = size_t(p.heads) * p.vdim_pad;
  float* out = p.out + size_t(first) * pitch + size_t(head) * p.vdim_pad + first_value;
#pragma unroll
  for (int n = 0; n < 8; ++n) {
    if (n * 8 < values) {
      if (lo_row < live) *reinterpret_cast<float2*>(out + size_t(lo_row) * pitch + n * 8 + 2 * c) = make_float2(acc[n][0], acc[n][1]);
      if (hi_row < live) *reinterpret_cast<float2*>(out + size_t(hi_row) * pitch + n * 8 + 2 * c) = make_float2(acc[n][2], acc[n][3]);
    }
  }
}

template <typename T, int kRows>
void launch_step_rows(const LightningParams& p, cudaStream_t stream, bool pdl) {
  static thread_local int configured_device = -1;
  int device = 0;
  EI_CUDA(cudaGetDevice(&device));
  if (configured_device != device) {
    EI_CUDA(cudaFuncSetAttribute(lightning_step_kernel<T, kRows>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                 int(step_shared_floats(kRows, kMaxHeadDim) * sizeof(float))));
    configured_device = device;
  }
  launch(lightning_step_kernel<T, kRows>, dim3(p.heads, p.vdim_pad / 16), dim3(kStepThreads),
         step_shared_floats(kRows, p.dim_pad) * sizeof(float), stream, pdl, p);
}

}  // namespace

template <typename T>
void launch_lightning_step(const LightningParams& p, cudaStream_t stream, bool pdl) {
  if (p.rows < 1 || p.rows > kPendingRows || p.dim_pad > kMaxHeadDim)
    throw std::invalid_argument("linear attention step takes 1..16 rows and key sizes up to 512");
  if (p.rows == 1) return launch_step_rows<T, 1>(p, stream, pdl);
  if (p.rows <= 4) return launch_step_rows<T, 4>(p, stream, pdl);
  return launch_step_rows<T, 16>(p, stream, pdl);
}
template void launch_lightning_step<float>(const LightningParams&, cudaStream_t, bool);
template void launch_lightning_step<bf16>(const LightningParams&, cudaStream_t, bool);

bool lightning_prompt_ok(int dim_pad, int vdim_pad) { return dim_pad <= 256 && dim_pad % 16 == 0 && vdim_pad % 16 == 0; }

namespace {
template <bool kToken>
void launch_prompt_kernels(const LightningParams& p, cudaStream_t stream, bool pdl) {
  static thread_local int configured_device = -1;
  int device = 0;
  EI_CUDA(cudaGetDevice(&device));
  if (configured_device != device) {
    EI_CUDA(cudaFuncSetAttribute(lightning_chunk_kernel<kToken>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(chunk_state_shared(256))));
    EI_CUDA(cudaFuncSetAttribute(lightning_output_kernel<kToken>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(output_shared(256))));
    configured_device = device;
  }
  const unsigned chunks = unsigned((p.rows + kChunk - 1) / kChunk), slices = unsigned((p.vdim_pad + kSlice - 1) / kSlice);
  const size_t quads = size_t(p.heads) * p.vdim_pad / 4 * p.dim_pad;
  launch(lightning_chunk_kernel<kToken>, dim3(chunks, p.heads, slices), dim3(kPromptThreads), chunk_state_shared(p.dim_pad), stream, pdl, p);
  launch(lightning_scan_kernel<kToken>, dim3(unsigned((quads + 255) / 256)), dim3(256), 0, stream, pdl, p);
  launch(lightning_output_kernel<kToken>, dim3(chunks, p.heads, slices), dim3(kPromptThreads), output_shared(p.dim_pad), stream, pdl, p);
}
}  // namespace

void launch_lightning_prompt(const LightningParams& p, cudaStream_t stream, bool pdl, int* launches) {
  if (!lightning_prompt_ok(p.dim_pad, p.vdim_pad)) throw std::invalid_argument("linear attention prompt takes key sizes up to 256");
  p.token.step ? launch_prompt_kernels<true>(p, stream, pdl) : launch_prompt_kernels<false>(p, stream, pdl);
  if (launches) *launches += 3;
}

}  // namespace ei
