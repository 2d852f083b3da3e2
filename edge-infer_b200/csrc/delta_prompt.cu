// The gated delta rule over a prompt, in chunks of 64 tokens.
//
// With G_t the cumulative logarithm of the decays inside a chunk (one per key channel), S the state ahead of it and u_t
// the vector that token t writes,
//   u_t = b_t (v_t - (k_t e^{G_t})^T S - sum_{j<t} A_tj u_j),   A_tj = sum_d k_t k_j e^{G_t - G_j}
//   out_t = (q_t e^{G_t})^T S + sum_{j<=t} B_tj u_j,            B_tj = sum_d q_t k_j e^{G_t - G_j}
// so with the unit lower triangular matrix L = I + diag(b) A the writes are U = V' - W S with V' = L^-1 diag(b) V and
// W = L^-1 diag(b) (k e^G), neither of which knows the state. The first kernel computes W, V', B and the scaled q and k of
// every chunk in parallel, the second walks the chunks with the state in registers.
//
// No exponent is ever positive: e^{G_t - G_j} is taken directly inside the 16 x 16 blocks on the diagonal, and through the
// end of the preceding block of 16, which lies between the two tokens, elsewhere. Everything is FP32 up to the operands of
// mma.sync, which enter as two BF16 terms (three products), and those are laid out in the order of its fragments, so the
// second kernel loads them straight from memory into registers.
#include "layered_device.cuh"

#include <algorithm>
#include <stdexcept>

namespace ei {
namespace {

constexpr int kChunk = kDeltaChunk;
constexpr int kBlock = 16;
constexpr int kThreads = 256;
constexpr int kPitchA = kChunk;       // floats per row of A transposed, read four at a time
constexpr int kPitchB = kChunk + 1;   // of B, written down its columns

// Places of one (chunk, head) in the chunk workspace, in bytes.
struct ChunkLayout {
  size_t w, q, k, b, v, decay, total;
};
__host__ __device__ inline ChunkLayout chunk_layout(int dim, int vdim) {
  ChunkLayout l{};
  const size_t operand = size_t(kChunk) * dim * 4;  // two BF16 terms per value
  l.w = 0;
  l.q = operand;
  l.k = 2 * operand;
  l.b = 3 * operand;
  l.v = l.b + size_t(kChunk) * kChunk * 4;
  l.decay = l.v + size_t(kChunk) * vdim * 4;
  l.total = (l.decay + size_t(dim) * 4 + 255) & ~size_t(255);
  return l;
}

size_t prepare_shared(int dim) {
  return (size_t(3) * kChunk * (dim + 1) + size_t(kChunk) * (kPitchA + kPitchB) + kChunk) * sizeof(float);
}

// Writes the A fragment of a 16 x 16 tile for this lane: values (g, 2c), (g, 2c+1), (g+8, ..), (g, 2c+8), .. in `x`.
__device__ __forceinline__ void store_fragment(uint4* to, const float (&x)[8]) {
  uint4 leading, rest;
  split_pair(x[0], x[1], leading.x, rest.x);
  split_pair(x[2], x[3], leading.y, rest.y);
  split_pair(x[4], x[5], leading.z, rest.z);
  split_pair(x[6], x[7], leading.w, rest.w);
  to[0] = leading;
  to[32] = rest;
}

__global__ void __launch_bounds__(kThreads) delta_chunk_kernel(const DeltaPromptParams p) {
  extern __shared__ __align__(16) float chunk_smem[];
  const OuterStateParams& o = p.outer;
  const int dim = o.dim_pad, pitch = dim + 1;
  float* at = chunk_smem;                          // diag(b) A transposed: at[j][t], j < t
  float* bm = at + kChunk * kPitchA;               // B: bm[t][j], j <= t
  float* beta = bm + kChunk * kPitchB;             // [kChunk]
  float* gs = beta + kChunk;                       // [kChunk][pitch]: cumulative logarithms of the decays
  float* ks = gs + kChunk * pitch;                 // [kChunk][pitch]: unit k, then columns of W
  float* qs = ks + kChunk * pitch;                 // [kChunk][pitch]: scaled unit q, then columns of V'
  grid_dependency_wait();
  grid_launch_dependents();
  const int context = o.control->context;
  if (context < 0 || context + o.rows > o.capacity) return;
  const int chunk = blockIdx.x, head = blockIdx.y, key_head = head / (o.heads / o.key_heads);
  const int first = chunk * kChunk, live = min(kChunk, o.rows - first);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
  const ChunkLayout layout = chunk_layout(dim, o.vdim_pad);
  unsigned char* own = p.chunks + (size_t(chunk) * o.heads + head) * layout.total;
  const bf16* conv = p.conv + size_t(first) * p.channels;
  const float* inverse = p.inverse + size_t(first) * 2 * o.key_heads;
  const float rate = o.rate[head];

  if (threadIdx.x < kChunk) {
    const int t = threadIdx.x;
    beta[t] = t < live ? sigmoid_value(__bfloat162float(static_cast<const bf16*>(o.fused)[size_t(first + t) * o.stride + o.step_at + head])) : 0.0f;
  }
  for (int i = threadIdx.x; i < kChunk * (dim / 2); i += kThreads) {
    const int t = i / (dim / 2), d = (i - t * (dim / 2)) * 2;
    float2 q = make_float2(0.0f, 0.0f), k = q, l = q;
    if (t < live) {
      const float q_scale = inverse[size_t(t) * 2 * o.key_heads + key_head], k_scale = inverse[size_t(t) * 2 * o.key_heads + o.key_heads + key_head];
      q = load_pair(conv + size_t(t) * p.channels + key_head * dim + d);
      k = load_pair(conv + size_t(t) * p.channels + (o.key_heads + key_head) * dim + d);
      q = make_float2(q.x * q_scale, q.y * q_scale);
      k = make_float2(k.x * k_scale, k.y * k_scale);
      const float2 a = load_pair(static_cast<const bf16*>(o.decay) + size_t(first + t) * o.decay_stride + head * dim + d);
      const float2 bias = load_pair(o.bias + head * dim + d);
      l = make_float2(-rate * softplus_value(a.x + bias.x), -rate * softplus_value(a.y + bias.y));
    }
    gs[t * pitch + d] = l.x;
    gs[t * pitch + d + 1] = l.y;
    ks[t * pitch + d] = k.x;
    ks[t * pitch + d + 1] = k.y;
    qs[t * pitch + d] = q.x;
    qs[t * pitch + d + 1] = q.y;
  }
  __syncthreads();
  // Cumulative sums: inside blocks of 16 rows, then the blocks' totals.
  for (int i = threadIdx.x; i < dim * (kChunk / kBlock); i += kThreads) {
    float* column = gs + (i / dim) * kBlock * pitch + i % dim;
    float sum = 0.0f;
#pragma unroll
    for (int t = 0; t < kBlock; ++t) column[t * pitch] = sum += column[t * pitch];
  }
  __syncthreads();
  for (int d = threadIdx.x; d < dim; d += kThreads) {
    for (int b = 1; b < kChunk / kBlock; ++b) {
      const float before = gs[(b * kBlock - 1) * pitch + d];
#pragma unroll
      for (int t = 0; t < kBlock; ++t) gs[(b * kBlock + t) * pitch + d] += before;
    }
  }
  __syncthreads();

  // A and B outside the diagonal blocks: tasks of 16 rows x 8 columns, through the end of the block ahead of the rows.
  for (int task = warp; task < 12; task += kThreads / 32) {
    const int block = task < 2 ? 1 : task < 6 ? 2 : 3, column = (task - (block == 1 ? 0 : block == 2 ? 2 : 6)) * 8;
    const int t0 = block * kBlock;
    const float* turn = gs + (t0 - 1) * pitch;
    float ka[4] = {0.0f, 0.0f, 0.0f, 0.0f}, qa[4] = {0.0f, 0.0f, 0.0f, 0.0f};
    for (int kk = 0; kk < dim / 16; ++kk) {
      uint32_t kh[4], kl[4], qh[4], ql[4], bh[2], bl[2];
#pragma unroll
      for (int part = 0; part < 4; ++part) {
        const int t = t0 + g + (part & 1) * 8, d = kk * 16 + 2 * c + (part >> 1) * 8;
        const float e0 = __expf(gs[t * pitch + d] - turn[d]), e1 = __expf(gs[t * pitch + d + 1] - turn[d + 1]);
        split_pair(ks[t * pitch + d] * e0, ks[t * pitch + d + 1] * e1, kh[part], kl[part]);
        split_pair(qs[t * pitch + d] * e0, qs[t * pitch + d + 1] * e1, qh[part], ql[part]);
      }
#pragma unroll
      for (int part = 0; part < 2; ++part) {
        const int j = column + g, d = kk * 16 + 2 * c + part * 8;
        split_pair(ks[j * pitch + d] * __expf(turn[d] - gs[j * pitch + d]), ks[j * pitch + d + 1] * __expf(turn[d + 1] - gs[j * pitch + d + 1]),
                   bh[part], bl[part]);
      }
      mma_bf16_16816(ka, kh[0], kh[1], kh[2], kh[3], bh[0], bh[1]);
      mma_bf16_16816(qa, qh[0], qh[1], qh[2], qh[3], bh[0], bh[1]);
      mma_bf16_16816(ka, kh[0], kh[1], kh[2], kh[3], bl[0], bl[1]);
      mma_bf16_16816(qa, qh[0], qh[1], qh[2], qh[3], bl[0], bl[1]);
      mma_bf16_16816(ka, kl[0], kl[1], kl[2], kl[3], bh[0], bh[1]);
      mma_bf16_16816(qa, ql[0], ql[1], ql[2], ql[3], bh[0], bh[1]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int t = t0 + g + (i >> 1) * 8, j = column + 2 * c + (i & 1);
      at[j * kPitchA + t] = ka[i] * beta[t];
      bm[t * kPitchB + j] = qa[i];
    }
  }
  // Inside the diagonal blocks: a thread per (row, column).
  for (int i = threadIdx.x; i < kChunk * kBlock; i += kThreads) {
    const int t = i & (kChunk - 1), j = (t & ~(kBlock - 1)) + (i >> 6);  // a warp's threads: rows one after the other
    float kk = 0.0f, qk = 0.0f;
    if (j <= t) {
      const float *gt = gs + t * pitch, *gj = gs + j * pitch, *kt = ks + t * pitch, *kj = ks + j * pitch, *qt = qs + t * pitch;
#pragma unroll 4
      for (int d = 0; d < dim; ++d) {
        const float x = kj[d] * __expf(gt[d] - gj[d]);
        kk = fmaf(kt[d], x, kk);
        qk = fmaf(qt[d], x, qk);
      }
    }
    at[j * kPitchA + t] = j < t ? kk * beta[t] : 0.0f;
    bm[t * kPitchB + j] = j <= t ? qk : 0.0f;
  }
  __syncthreads();

  // Operands that need no solving: q e^G, k e^(G_end - G) transposed, B, and the chunk's decay.
  const float* last = gs + (kChunk - 1) * pitch;
  uint4* q_out = reinterpret_cast<uint4*>(own + layout.q);
  uint4* k_out = reinterpret_cast<uint4*>(own + layout.k);
  uint4* b_out = reinterpret_cast<uint4*>(own + layout.b);
  const int steps = dim / 16;
  for (int tile = warp; tile < 4 * steps; tile += kThreads / 32) {
    const int mt = tile / steps, kk = tile - mt * steps;
    float x[8], y[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const int row = g + ((e >> 1) & 1) * 8, col = 2 * c + (e & 1) + (e >> 2) * 8;
      const int t = mt * 16 + row, d = kk * 16 + col;
      x[e] = qs[t * pitch + d] * __expf(gs[t * pitch + d]);
      // Tile (kk, mt) of the transpose: rows are key channels, columns tokens.
      const int token = mt * 16 + col, channel = kk * 16 + row;
      y[e] = ks[token * pitch + channel] * __expf(last[channel] - gs[token * pitch + channel]);
    }
    store_fragment(q_out + size_t(mt * steps + kk) * 64 + lane, x);
    store_fragment(k_out + size_t(kk * 4 + mt) * 64 + lane, y);
  }
  for (int tile = warp; tile < 16; tile += kThreads / 32) {
    const int mt = tile >> 2, kk = tile & 3;
    if (kk > mt) continue;
    float x[8];
#pragma unroll
    for (int e = 0; e < 8; ++e)
      x[e] = bm[(mt * 16 + g + ((e >> 1) & 1) * 8) * kPitchB + kk * 16 + 2 * c + (e & 1) + (e >> 2) * 8];
    store_fragment(b_out + size_t(tile) * 64 + lane, x);
  }
  for (int d = threadIdx.x; d < dim; d += kThreads) reinterpret_cast<float*>(own + layout.decay)[d] = __expf(last[d]);
  __syncthreads();

  // Solves (I + diag(b) A) X = right-hand side for one column in place, 16 rows at a time.
  auto solve = [&](float* column) {
#pragma unroll 1
    for (int b = 0; b < kChunk / kBlock; ++b) {
      float x[kBlock];
#pragma unroll
      for (int i = 0; i < kBlock; ++i) x[i] = column[(b * kBlock + i) * pitch];
#pragma unroll 2
      for (int j = 0; j < b * kBlock; ++j) {
        const float known = column[j * pitch];
        const float* a = at + j * kPitchA + b * kBlock;
#pragma unroll
        for (int i = 0; i < kBlock; i += 4) {
          const float4 v = *reinterpret_cast<const float4*>(a + i);
          x[i] = fmaf(-v.x, known, x[i]);
          x[i + 1] = fmaf(-v.y, known, x[i + 1]);
          x[i + 2] = fmaf(-v.z, known, x[i + 2]);
          x[i + 3] = fmaf(-v.w, known, x[i + 3]);
        }
      }
#pragma unroll
      for (int j = 0; j < kBlock - 1; ++j) {
        const float* a = at + (b * kBlock + j) * kPitchA + b * kBlock;
#pragma unroll
        for (int i = (j + 1) & ~3; i < kBlock; i += 4) {
          const float4 v = *reinterpret_cast<const float4*>(a + i);  // zero up to the diagonal
          x[i] = i > j ? fmaf(-v.x, x[j], x[i]) : x[i];
          x[i + 1] = i + 1 > j ? fmaf(-v.y, x[j], x[i + 1]) : x[i + 1];
          x[i + 2] = i + 2 > j ? fmaf(-v.z, x[j], x[i + 2]) : x[i + 2];
          x[i + 3] = i + 3 > j ? fmaf(-v.w, x[j], x[i + 3]) : x[i + 3];
        }
      }
#pragma unroll
      for (int i = 0; i < kBlock; ++i) column[(b * kBlock + i) * pitch] = x[i];
    }
  };
  // The columns of W in place of k, those of V' in place of q, `dim` value columns at a time.
  float4* v_out = reinterpret_cast<float4*>(own + layout.v);
  const bf16* values = conv + 2 * o.key_heads * dim + head * o.vdim_pad;
  for (int v0 = 0; v0 < o.vdim_pad; v0 += dim) {
    const int width = min(dim, o.vdim_pad - v0);
    for (int i = threadIdx.x; i < kChunk * (width / 2); i += kThreads) {
      const int t = i / (width / 2), d = (i - t * (width / 2)) * 2;
      const float2 v = t < live ? load_pair(values + size_t(t) * p.channels + v0 + d) : make_float2(0.0f, 0.0f);
      qs[t * pitch + d] = v.x * beta[t];
      qs[t * pitch + d + 1] = v.y * beta[t];
    }
    __syncthreads();
    const int unsolved = v0 == 0 ? dim : 0;  // columns of W still to come, ahead of the value columns
    for (int column = threadIdx.x; column < unsolved + width; column += kThreads) {
      if (column < unsolved) {
#pragma unroll 4
        for (int t = 0; t < kChunk; ++t) ks[t * pitch + column] *= beta[t] * __expf(gs[t * pitch + column]);
        solve(ks + column);
      } else {
        solve(qs + column - unsolved);
      }
    }
    __syncthreads();
    // V' in the order of the accumulators: [row tile][column tile of 8][lane].
    for (int tile = warp; tile < 4 * (width / 8); tile += kThreads / 32) {
      const int mt = tile / (width / 8), nt = tile - mt * (width / 8);
      const float* x = qs + (mt * 16 + g) * pitch + nt * 8 + 2 * c;
      v_out[(size_t(mt) * (o.vdim_pad / 8) + v0 / 8 + nt) * 32 + lane] = make_float4(x[0], x[1], x[8 * pitch], x[8 * pitch + 1]);
    }
    __syncthreads();
  }
  uint4* w_out = reinterpret_cast<uint4*>(own + layout.w);
  for (int tile = warp; tile < 4 * steps; tile += kThreads / 32) {
    const int mt = tile / steps, kk = tile - mt * steps;
    float x[8];
#pragma unroll
    for (int e = 0; e < 8; ++e)
      x[e] = ks[(mt * 16 + g + ((e >> 1) & 1) * 8) * pitch + kk * 16 + 2 * c + (e & 1) + (e >> 2) * 8];
    store_fragment(w_out + size_t(tile) * 64 + lane, x);
  }
}

// Block (head, kColumns values), eight warps, the chunks one after the other. Warps 0-3 hold 16 rows each of U, warps 4-7
// of the output; every warp holds kTiles tiles of 16 key channels of the state.
template <int kColumns, int kTiles>
__global__ void __launch_bounds__(kThreads) delta_scan_kernel(const DeltaPromptParams p) {
  constexpr int kN = kColumns / 8;              // accumulator tiles per row tile
  constexpr int kPitch = kColumns + 8;          // BF16 elements per staged row: an odd number of 16-byte pieces
  extern __shared__ __align__(16) unsigned char scan_smem[];
  const OuterStateParams& o = p.outer;
  const int dim = o.dim_pad, steps = dim / 16;
  bf16* state_leading = reinterpret_cast<bf16*>(scan_smem);       // [dim][kPitch]
  bf16* state_rest = state_leading + dim * kPitch;
  bf16* write_leading = state_rest + dim * kPitch;                // [kChunk][kPitch]
  bf16* write_rest = write_leading + kChunk * kPitch;
  grid_dependency_wait();
  grid_launch_dependents();
  const int context = o.control->context, base = o.control->state_base;
  if (context < 0 || context + o.rows > o.capacity) return;
  const int pending = min(kPendingRows, max(0, context - base));
  const int head = blockIdx.x, first_value = blockIdx.y * kColumns, key_head = head / (o.heads / o.key_heads);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
  const int matrix = lane >> 3, in_matrix = lane & 7;
  const ChunkLayout layout = chunk_layout(dim, o.vdim_pad);
  const int chunks = (o.rows + kChunk - 1) / kChunk;
  const int live_columns = min(kColumns, o.vdim_pad - first_value);  // a multiple of 16

  // The state as accumulators: rows are key channels; pending rows folded in.
  float s[kTiles][kN][4];
  auto state_at = [&](int d, int n) {  // address of values n, n + 1 (even n) of key channel d
    const int v = first_value + n;
    return o.state + ((size_t(head) * (o.vdim_pad / 16) + v / 16) * dim + d) * 16 + (v & 15);
  };
#pragma unroll
  for (int m = 0; m < kTiles; ++m) {
    const int tile = warp + 8 * m;
#pragma unroll
    for (int n = 0; n < kN; ++n) {
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int d = tile * 16 + g + half * 8, col = n * 8 + 2 * c;
        float2 x = make_float2(0.0f, 0.0f);
        if (tile < steps && col < live_columns) {
          if (base > 0) x = *reinterpret_cast<const float2*>(state_at(d, col));
          for (int j = 0; j < pending; ++j) {
            const size_t slot = (base + j) & (kRingRows - 1);
            const float k = o.ring_k[(slot * o.key_heads + key_head) * dim + d], decay = o.ring_g[(slot * o.heads + head) * dim + d];
            const float2 u = *reinterpret_cast<const float2*>(o.ring_u + (slot * o.heads + head) * o.vdim_pad + first_value + col);
            x = make_float2(fmaf(k, u.x, decay * x.x), fmaf(k, u.y, decay * x.y));
          }
        }
        s[m][n][2 * half] = x.x;
        s[m][n][2 * half + 1] = x.y;
      }
    }
  }
  auto publish = [&](const float (&x)[kN][4], int row, bf16* leading, bf16* rest) {
#pragma unroll
    for (int n = 0; n < kN; ++n) {
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t hi, lo;
        split_pair(x[n][2 * half], x[n][2 * half + 1], hi, lo);
        const int at = (row + g + half * 8) * kPitch + n * 8 + 2 * c;
        *reinterpret_cast<uint32_t*>(leading + at) = hi;
        *reinterpret_cast<uint32_t*>(rest + at) = lo;
      }
    }
  };
#pragma unroll
  for (int m = 0; m < kTiles; ++m)
    if (warp + 8 * m < steps) publish(s[m], (warp + 8 * m) * 16, state_leading, state_rest);
  __syncthreads();

  // acc += (two-term A fragment) x (two-term rows of `leading` / `rest` from `row` on).
  auto multiply = [&](float (&acc)[kN][4], const uint4& ah, const uint4& al, const bf16* leading, const bf16* rest, int row) {
#pragma unroll
    for (int n = 0; n < kN; n += 2) {
      const int at = (row + (matrix & 1) * 8 + in_matrix) * kPitch + (n + (matrix >> 1)) * 8;
      uint32_t b0, b1, b2, b3;
      ldmatrix_x4_trans(b0, b1, b2, b3, leading + at);
      mma_bf16_16816(acc[n], ah.x, ah.y, ah.z, ah.w, b0, b1);
      mma_bf16_16816(acc[n + 1], ah.x, ah.y, ah.z, ah.w, b2, b3);
      mma_bf16_16816(acc[n], al.x, al.y, al.z, al.w, b0, b1);
      mma_bf16_16816(acc[n + 1], al.x, al.y, al.z, al.w, b2, b3);
      ldmatrix_x4_trans(b0, b1, b2, b3, rest + at);
      mma_bf16_16816(acc[n], ah.x, ah.y, ah.z, ah.w, b0, b1);
      mma_bf16_16816(acc[n + 1], ah.x, ah.y, ah.z, ah.w, b2, b3);
    }
  };
  constexpr int kAhead = 8;  // K steps of an operand requested at once
  const int row_tile = warp & 3;
  for (int chunk = 0; chunk < chunks; ++chunk) {
    const unsigned char* own = p.chunks + (size_t(chunk) * o.heads + head) * layout.total;
    const uint4* operand = reinterpret_cast<const uint4*>(own + (warp < 4 ? layout.w : layout.q)) + size_t(row_tile) * steps * 64 + lane;
    float acc[kN][4];
#pragma unroll
    for (int n = 0; n < kN; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.0f;
    for (int kk = 0; kk < steps; kk += kAhead) {
      uint4 ah[kAhead], al[kAhead];
#pragma unroll
      for (int i = 0; i < kAhead; ++i) {
        if (kk + i < steps) {
          ah[i] = operand[size_t(kk + i) * 64];
          al[i] = operand[size_t(kk + i) * 64 + 32];
        }
      }
#pragma unroll
      for (int i = 0; i < kAhead; ++i)
        if (kk + i < steps) multiply(acc, ah[i], al[i], state_leading, state_rest, (kk + i) * 16);
    }
    if (warp < 4) {
      const float4* v = reinterpret_cast<const float4*>(own + layout.v) + (size_t(row_tile) * (o.vdim_pad / 8) + first_value / 8) * 32 + lane;
#pragma unroll
      for (int n = 0; n < kN; ++n) {
        const float4 x = n * 8 < live_columns ? v[n * 32] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        acc[n][0] = x.x - acc[n][0];
        acc[n][1] = x.y - acc[n][1];
        acc[n][2] = x.z - acc[n][2];
        acc[n][3] = x.w - acc[n][3];
      }
      publish(acc, row_tile * 16, write_leading, write_rest);
    }
    __syncthreads();  // the writes are there, and every warp is done with the staged state
    const uint4* keys = reinterpret_cast<const uint4*>(own + layout.k) + lane;
    const float* decay = reinterpret_cast<const float*>(own + layout.decay);
#pragma unroll
    for (int m = 0; m < kTiles; ++m) {
      const int tile = warp + 8 * m;
      if (tile >= steps) break;
      uint4 ah[4], al[4];
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        ah[kk] = keys[size_t(tile * 4 + kk) * 64];
        al[kk] = keys[size_t(tile * 4 + kk) * 64 + 32];
      }
      const float lo = decay[tile * 16 + g], hi = decay[tile * 16 + g + 8];
#pragma unroll
      for (int n = 0; n < kN; ++n) {
        s[m][n][0] *= lo;
        s[m][n][1] *= lo;
        s[m][n][2] *= hi;
        s[m][n][3] *= hi;
      }
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) multiply(s[m], ah[kk], al[kk], write_leading, write_rest, kk * 16);
      publish(s[m], tile * 16, state_leading, state_rest);
    }
    if (warp >= 4) {
      const uint4* inside = reinterpret_cast<const uint4*>(own + layout.b) + size_t(row_tile) * 4 * 64 + lane;
      for (int kk = 0; kk <= row_tile; ++kk) multiply(acc, inside[size_t(kk) * 64], inside[size_t(kk) * 64 + 32], write_leading, write_rest, kk * 16);
      const int row = chunk * kChunk + row_tile * 16 + g;
      const size_t out_pitch = size_t(o.heads) * o.vdim_pad;
      float* out = o.out + size_t(row) * out_pitch + head * o.vdim_pad + first_value + 2 * c;
#pragma unroll
      for (int n = 0; n < kN; ++n) {
        if (n * 8 >= live_columns) continue;
        if (row < o.rows) *reinterpret_cast<float2*>(out + n * 8) = make_float2(acc[n][0], acc[n][1]);
        if (row + 8 < o.rows) *reinterpret_cast<float2*>(out + 8 * out_pitch + n * 8) = make_float2(acc[n][2], acc[n][3]);
      }
    }
    __syncthreads();  // the next state is there, and every warp is done with the writes
  }
#pragma unroll
  for (int m = 0; m < kTiles; ++m) {
    const int tile = warp + 8 * m;
    if (tile >= steps) break;
#pragma unroll
    for (int n = 0; n < kN; ++n) {
      if (n * 8 >= live_columns) continue;
      *reinterpret_cast<float2*>(state_at(tile * 16 + g, n * 8 + 2 * c)) = make_float2(s[m][n][0], s[m][n][1]);
      *reinterpret_cast<float2*>(state_at(tile * 16 + g + 8, n * 8 + 2 * c)) = make_float2(s[m][n][2], s[m][n][3]);
    }
  }
}

size_t scan_shared(int dim, int columns) { return size_t(2) * (dim + kChunk) * (columns + 8) * 2; }

template <int kColumns, int kTiles>
void launch_scan(const DeltaPromptParams& p, cudaStream_t stream, bool pdl) {
  static thread_local int configured_device = -1;
  int device = 0;
  EI_CUDA(cudaGetDevice(&device));
  if (configured_device != device) {
    EI_CUDA(cudaFuncSetAttribute(delta_scan_kernel<kColumns, kTiles>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                 int(scan_shared(256, kColumns))));
    configured_device = device;
  }
  launch(delta_scan_kernel<kColumns, kTiles>, dim3(unsigned(p.outer.heads), unsigned((p.outer.vdim_pad + kColumns - 1) / kColumns)),
         dim3(kThreads), scan_shared(p.outer.dim_pad, kColumns), stream, pdl, p);
}

}  // namespace

bool delta_prompt_ok(int dim_pad, int vdim_pad) { return dim_pad <= 256 && dim_pad % 16 == 0 && vdim_pad % 16 == 0; }

size_t delta_prompt_bytes(size_t rows, size_t heads, size_t dim_pad, size_t vdim_pad) {
  return (rows + kChunk - 1) / kChunk * heads * chunk_layout(int(dim_pad), int(vdim_pad)).total;
}

void launch_delta_prompt(const DeltaPromptParams& p, cudaStream_t stream, bool pdl) {
  if (!delta_prompt_ok(p.outer.dim_pad, p.outer.vdim_pad)) throw std::invalid_argument("the delta rule's prompt form takes key sizes up to 256");
  static thread_local int configured_device = -1;
  static thread_local int multiprocessors = 1;
  int device = 0;
  EI_CUDA(cudaGetDevice(&device));
  if (configured_device != device) {
    EI_CUDA(cudaDeviceGetAttribute(&multiprocessors, cudaDevAttrMultiProcessorCount, device));
    EI_CUDA(cudaFuncSetAttribute(delta_chunk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(prepare_shared(256))));
    configured_device = device;
  }
  const unsigned chunks = unsigned((p.outer.rows + kChunk - 1) / kChunk);
  launch(delta_chunk_kernel, dim3(chunks, unsigned(p.outer.heads)), dim3(kThreads), prepare_shared(p.outer.dim_pad), stream, pdl, p);
  // Narrow blocks where wide ones would leave most of the chip idle.
  const bool narrow = p.outer.heads * ((p.outer.vdim_pad + 31) / 32) * 3 < multiprocessors * 2;
  if (p.outer.dim_pad <= 128)
    return narrow ? launch_scan<16, 1>(p, stream, pdl) : launch_scan<32, 1>(p, stream, pdl);
  narrow ? launch_scan<16, 2>(p, stream, pdl) : launch_scan<32, 2>(p, stream, pdl);
}

}  // namespace ei
