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

// Floats per staged row: sixteen more than a multiple of 32 keeps four-value accesses of two rows apart in the banks.
__host__ __device__ inline int row_pitch(int dim) {
  if (dim > 192) return dim < 256 ? dim + 4 : dim;  // what shared memory has room for
  if (dim < 48) return 48;  // the decays' place holds ten 16 x 16 matrices later
  return dim % 32 == 16 ? dim : dim + 16;
}
size_t prepare_shared(int dim) {
  return (size_t(3) * kChunk * row_pitch(dim) + size_t(kChunk) * (kPitchA + kPitchB) + kChunk) * sizeof(float);
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
// The same from four consecutive values of row g and of row g + 8: columns 4 c .. 4 c + 3 of the tile stand where the
// fragment has 2 c, 2 c + 1, 2 c + 8, 2 c + 9. Both operands of a product use this order, so the sum is the same.
__device__ __forceinline__ void store_fragment(uint4* to, float4 lo, float4 hi) {
  const float x[8] = {lo.x, lo.y, hi.x, hi.y, lo.z, lo.w, hi.z, hi.w};
  store_fragment(to, x);
}
// Where tokens are summed over, value e of lane c's fragment belongs to this token of the tile's 16 (of both operands).
__device__ __forceinline__ int token_of(int c, int e) { return c + 4 * (e & 1) + 8 * (e >> 2); }
// Its place among the operand's rows, from the token.
__device__ __forceinline__ int token_place(int t) { return 2 * (t & 3) + ((t >> 2) & 1) + 8 * (t >> 3); }
__device__ __forceinline__ float4 quad_at(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 times(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }
// The decays' logarithms are kept to base two.
__device__ __forceinline__ float power_of_two(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float4 exp_of(float4 a) { return make_float4(power_of_two(a.x), power_of_two(a.y), power_of_two(a.z), power_of_two(a.w)); }
__device__ __forceinline__ float4 minus(float4 a, float4 b) { return make_float4(a.x - b.x, a.y - b.y, a.z - b.z, a.w - b.w); }
__device__ __forceinline__ float4 exp_between(float4 a, float4 b) { return exp_of(minus(a, b)); }
// The same for a difference that may be above zero where the result is not used: held at zero so that it stays finite.
__device__ __forceinline__ float4 exp_below(float4 a, float4 b) {
  const float4 x = minus(a, b);
  return exp_of(make_float4(fminf(x.x, 0.0f), fminf(x.y, 0.0f), fminf(x.z, 0.0f), fminf(x.w, 0.0f)));
}
__device__ __forceinline__ float dot(float4 a, float4 b, float sum) {
  return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, sum))));
}
// A operand registers (leading, rest) of rows g and g + 8 in that order, and B operand registers of one row.
__device__ __forceinline__ void split_rows(float4 lo, float4 hi, uint32_t (&leading)[4], uint32_t (&rest)[4]) {
  split_pair(lo.x, lo.y, leading[0], rest[0]);
  split_pair(hi.x, hi.y, leading[1], rest[1]);
  split_pair(lo.z, lo.w, leading[2], rest[2]);
  split_pair(hi.z, hi.w, leading[3], rest[3]);
}

// Sixteen warps. Of A and B, warp w takes columns of a diagonal block and one tile below the diagonal.
constexpr int kPrepareThreads = 512;
__global__ void __launch_bounds__(kPrepareThreads) delta_chunk_kernel(const DeltaPromptParams p) {
  extern __shared__ __align__(16) float chunk_smem[];
  const OuterStateParams& o = p.outer;
  const int dim = o.dim_pad, pitch = row_pitch(dim), steps = dim / 16;
  float* at = chunk_smem;                          // diag(b) A transposed: at[j][t], j < t
  float* gs = at + kChunk * kPitchA;               // [kChunk][pitch]: cumulative logarithms of the decays
  float* ks = gs + kChunk * pitch;                 // [kChunk][pitch]: unit k, then columns of V'
  float* qs = ks + kChunk * pitch;                 // [kChunk][pitch]: scaled unit q, then columns of W
  float* bm = qs + kChunk * pitch;                 // B: bm[t][j], j <= t
  float* beta = bm + kChunk * kPitchB;             // [kChunk]
  grid_dependency_wait();
  grid_launch_dependents();
  const int context = o.control->context;
  if (context < 0 || context + o.rows > o.capacity) return;
  const int chunk = blockIdx.x, head = blockIdx.y, key_head = head / (o.heads / o.key_heads);
  const int first = chunk * kChunk, live = min(kChunk, o.rows - first);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
  constexpr int kWarps = kPrepareThreads / 32;
  const ChunkLayout layout = chunk_layout(dim, o.vdim_pad);
  unsigned char* own = p.chunks + (size_t(chunk) * o.heads + head) * layout.total;
  const bf16* conv = p.conv + size_t(first) * p.channels;
  const float* inverse = p.inverse + size_t(first) * 2 * o.key_heads;
  const float rate = o.rate[head] * 1.44269504f;  // logarithms to base two

  if (threadIdx.x < kChunk) {
    const int t = threadIdx.x;
    beta[t] = t < live ? sigmoid_value(__bfloat162float(static_cast<const bf16*>(o.fused)[size_t(first + t) * o.stride + o.step_at + head])) : 0.0f;
  }
  const int quads = dim / 4;
#pragma unroll 4
  for (int i = threadIdx.x; i < kChunk * quads; i += kPrepareThreads) {
    const int t = i / quads, d = (i - t * quads) * 4;
    float4 q = make_float4(0.0f, 0.0f, 0.0f, 0.0f), k = q, l = q;
    if (t < live) {
      const float q_scale = inverse[size_t(t) * 2 * o.key_heads + key_head], k_scale = inverse[size_t(t) * 2 * o.key_heads + o.key_heads + key_head];
      q = load_quad(conv + size_t(t) * p.channels + key_head * dim + d);
      k = load_quad(conv + size_t(t) * p.channels + (o.key_heads + key_head) * dim + d);
      l = add(load_quad(static_cast<const bf16*>(o.decay) + size_t(first + t) * o.decay_stride + head * dim + d),
              quad_at(o.bias + head * dim + d));
      q = make_float4(q.x * q_scale, q.y * q_scale, q.z * q_scale, q.w * q_scale);
      k = make_float4(k.x * k_scale, k.y * k_scale, k.z * k_scale, k.w * k_scale);
      l = make_float4(-rate * quick_softplus(l.x), -rate * quick_softplus(l.y), -rate * quick_softplus(l.z), -rate * quick_softplus(l.w));
    }
    *reinterpret_cast<float4*>(gs + t * pitch + d) = l;
    *reinterpret_cast<float4*>(ks + t * pitch + d) = k;
    *reinterpret_cast<float4*>(qs + t * pitch + d) = q;
  }
  __syncthreads();
  // Cumulative sums: inside blocks of 16 rows, then the blocks' totals.
  for (int i = threadIdx.x; i < dim * (kChunk / kBlock); i += kPrepareThreads) {
    float* column = gs + (i / dim) * kBlock * pitch + i % dim;
    float sum = 0.0f, x[kBlock];
#pragma unroll
    for (int t = 0; t < kBlock; ++t) x[t] = column[t * pitch];
#pragma unroll
    for (int t = 0; t < kBlock; ++t) column[t * pitch] = sum += x[t];
  }
  __syncthreads();
  for (int i = threadIdx.x; i < dim; i += kPrepareThreads) {
    float before[kChunk / kBlock];
    before[0] = 0.0f;
#pragma unroll
    for (int b = 1; b < kChunk / kBlock; ++b) before[b] = before[b - 1] + gs[(b * kBlock - 1) * pitch + i];
#pragma unroll
    for (int b = 1; b < kChunk / kBlock; ++b) {
      float x[kBlock];
#pragma unroll
      for (int t = 0; t < kBlock; ++t) x[t] = gs[(b * kBlock + t) * pitch + i];
#pragma unroll
      for (int t = 0; t < kBlock; ++t) gs[(b * kBlock + t) * pitch + i] = x[t] + before[b];
    }
  }
  __syncthreads();

  // The value columns are requested now and used after A and B.
  float4* v_out = reinterpret_cast<float4*>(own + layout.v);
  const bf16* values = conv + 2 * o.key_heads * dim + head * o.vdim_pad;
  constexpr int kValueQuads = 4;  // per thread: 64 rows of 128 values
  uint2 ahead[kValueQuads];
  const int first_width = min(dim, o.vdim_pad), first_quads = first_width / 4;
#pragma unroll
  for (int n = 0; n < kValueQuads; ++n) {
    const int i = threadIdx.x + n * kPrepareThreads, t = i / first_quads;
    ahead[n] = make_uint2(0, 0);
    if (t < live && t < kChunk) ahead[n] = *reinterpret_cast<const uint2*>(values + size_t(t) * p.channels + (i - t * first_quads) * 4);
  }

  // A and B inside the 8 x 8 blocks on the diagonal, directly. Warp w: row g of both blocks of the 16 x 16 block w >> 2
  // against columns 2 (w & 3), + 1 of its own block.
  {
    const int base = (warp >> 2) * kBlock, column = base + (warp & 3) * 2, t = base + g;
    float ka[2][2], qa[2][2];  // [early block, late block][column]
#pragma unroll
    for (int n = 0; n < 2; ++n) ka[n][0] = ka[n][1] = qa[n][0] = qa[n][1] = 0.0f;
#pragma unroll 2
    for (int d = 4 * c; d < dim; d += 16) {
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        const float4 gt = quad_at(gs + (t + 8 * n) * pitch + d), kt = quad_at(ks + (t + 8 * n) * pitch + d), qt = quad_at(qs + (t + 8 * n) * pitch + d);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int j = (column + e + 8 * n) * pitch + d;
          const float4 x = times(quad_at(ks + j), exp_below(gt, quad_at(gs + j)));
          ka[n][e] = dot(kt, x, ka[n][e]);
          qa[n][e] = dot(qt, x, qa[n][e]);
        }
      }
    }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        ka[n][e] += __shfl_xor_sync(0xffffffffu, ka[n][e], 1);
        ka[n][e] += __shfl_xor_sync(0xffffffffu, ka[n][e], 2);
        qa[n][e] += __shfl_xor_sync(0xffffffffu, qa[n][e], 1);
        qa[n][e] += __shfl_xor_sync(0xffffffffu, qa[n][e], 2);
      }
    // The four lanes of a row hold the same sums: lane c writes column c & 1 of block c >> 1, and B's zeros beside it.
    const float k_sum = c & 2 ? (c & 1 ? ka[1][1] : ka[1][0]) : (c & 1 ? ka[0][1] : ka[0][0]);
    const float q_sum = c & 2 ? (c & 1 ? qa[1][1] : qa[1][0]) : (c & 1 ? qa[0][1] : qa[0][0]);
    const int row = t + (c & 2) * 4, j = column + (c & 1) + (c & 2) * 4;
    at[j * kPitchA + row] = j < row ? k_sum * beta[row] : 0.0f;
    bm[row * kPitchB + j] = j <= row ? q_sum : 0.0f;
    if (c < 2) bm[t * kPitchB + column + c + 8] = 0.0f;
  }
  // Everything else below the diagonal, through the end of the block ahead of the rows: twelve tiles of 16 rows x 8 columns
  // below the 16 x 16 blocks, four of 8 x 8 inside them (rows g + 8 of those are not there).
  {
    const bool inside = warp >= 12;
    const int block = inside ? warp - 12 : warp < 2 ? 1 : warp < 6 ? 2 : 3;
    const int t0 = block * kBlock + (inside ? 8 : 0);
    const int column = inside ? block * kBlock : (warp - (block == 1 ? 0 : block == 2 ? 2 : 6)) * 8;
    const int high = inside ? 0 : 8;
    float ka[3][4], qa[3][4];  // a chain per product of terms
#pragma unroll
    for (int n = 0; n < 3; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) ka[n][e] = qa[n][e] = 0.0f;
#pragma unroll 2
    for (int d = 4 * c; d < dim; d += 16) {
      const float4 turn = quad_at(gs + (t0 - 1) * pitch + d);
      const int lo = (t0 + g) * pitch + d, hi = lo + high * pitch;
      const float4 e_lo = exp_between(quad_at(gs + lo), turn), e_hi = exp_between(quad_at(gs + hi), turn);
      uint32_t kh[4], kl[4], qh[4], ql[4], bh[2], bl[2];
      split_rows(times(quad_at(ks + lo), e_lo), times(quad_at(ks + hi), e_hi), kh, kl);
      split_rows(times(quad_at(qs + lo), e_lo), times(quad_at(qs + hi), e_hi), qh, ql);
      const float4 x = times(quad_at(ks + (column + g) * pitch + d), exp_between(turn, quad_at(gs + (column + g) * pitch + d)));
      split_pair(x.x, x.y, bh[0], bl[0]);
      split_pair(x.z, x.w, bh[1], bl[1]);
      mma_bf16_16816(ka[0], kh[0], kh[1], kh[2], kh[3], bh[0], bh[1]);
      mma_bf16_16816(qa[0], qh[0], qh[1], qh[2], qh[3], bh[0], bh[1]);
      mma_bf16_16816(ka[1], kh[0], kh[1], kh[2], kh[3], bl[0], bl[1]);
      mma_bf16_16816(qa[1], qh[0], qh[1], qh[2], qh[3], bl[0], bl[1]);
      mma_bf16_16816(ka[2], kl[0], kl[1], kl[2], kl[3], bh[0], bh[1]);
      mma_bf16_16816(qa[2], ql[0], ql[1], ql[2], ql[3], bh[0], bh[1]);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      if (e >= 2 && inside) break;
      const int t = t0 + g + (e >> 1) * 8, j = column + 2 * c + (e & 1);
      at[j * kPitchA + t] = (ka[0][e] + (ka[1][e] + ka[2][e])) * beta[t];
      bm[t * kPitchB + j] = qa[0][e] + (qa[1][e] + qa[2][e]);
    }
  }
  __syncthreads();

  // Operands that need no solving: q e^G, k e^(G_end - G) transposed, B, and the chunk's decay. A place of q that has been
  // read takes the right-hand side of W, b k e^G.
  const float* last = gs + (kChunk - 1) * pitch;
  uint4* q_out = reinterpret_cast<uint4*>(own + layout.q);
  uint4* k_out = reinterpret_cast<uint4*>(own + layout.k);
  uint4* b_out = reinterpret_cast<uint4*>(own + layout.b);
#pragma unroll 2
  for (int tile = warp; tile < 4 * steps; tile += kWarps) {
    const int mt = tile / steps, kk = tile - mt * steps;
    const int t = mt * 16 + g, lo = t * pitch + kk * 16 + 4 * c, hi = lo + 8 * pitch;
    const float4 e_lo = exp_of(quad_at(gs + lo)), e_hi = exp_of(quad_at(gs + hi));
    store_fragment(q_out + size_t(mt * steps + kk) * 64 + lane, times(quad_at(qs + lo), e_lo), times(quad_at(qs + hi), e_hi));
    const float b_lo = beta[t], b_hi = beta[t + 8];
    *reinterpret_cast<float4*>(qs + lo) = times(quad_at(ks + lo), make_float4(e_lo.x * b_lo, e_lo.y * b_lo, e_lo.z * b_lo, e_lo.w * b_lo));
    *reinterpret_cast<float4*>(qs + hi) = times(quad_at(ks + hi), make_float4(e_hi.x * b_hi, e_hi.y * b_hi, e_hi.z * b_hi, e_hi.w * b_hi));
    float y[8];  // tile (kk, mt) of the transpose: rows are key channels, columns tokens in the order of token_of
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const int token = mt * 16 + token_of(c, e), channel = kk * 16 + g + ((e >> 1) & 1) * 8;
      y[e] = ks[token * pitch + channel] * power_of_two(last[channel] - gs[token * pitch + channel]);
    }
    store_fragment(k_out + size_t(kk * 4 + mt) * 64 + lane, y);
  }
  for (int tile = warp; tile < 16; tile += kWarps) {
    const int mt = tile >> 2, kk = tile & 3;
    if (kk > mt) continue;
    float x[8];
#pragma unroll
    for (int e = 0; e < 8; ++e)
      x[e] = bm[(mt * 16 + g + ((e >> 1) & 1) * 8) * kPitchB + kk * 16 + token_of(c, e)];
    store_fragment(b_out + size_t(tile) * 64 + lane, x);
  }
  for (int d = threadIdx.x; d < dim; d += kPrepareThreads) reinterpret_cast<float*>(own + layout.decay)[d] = power_of_two(last[d]);
  // The inverses of the four unit lower triangular diagonal blocks, one column per thread, into the unused half of the
  // blocks' places: inverse[i][j], j < i, at at[16 b + i][16 b + j].
  if (threadIdx.x < kChunk) {
    const int base = threadIdx.x & ~(kBlock - 1), j = threadIdx.x & (kBlock - 1);
    float x[kBlock];
#pragma unroll
    for (int i = 0; i < kBlock; ++i) x[i] = i == j ? 1.0f : 0.0f;
#pragma unroll
    for (int m = 0; m < kBlock - 1; ++m)
#pragma unroll
      for (int i = m + 1; i < kBlock; ++i) x[i] = fmaf(-at[(base + m) * kPitchA + base + i], x[m], x[i]);
#pragma unroll
    for (int i = 1; i < kBlock; ++i)
      if (i > j) at[(base + i) * kPitchA + base + j] = x[i];
  }
  __syncthreads();

  // Solves (I + diag(b) A) X = right-hand side for the columns of W (in q's place) and of V' (in k's place) by blocks of 16
  // rows: X_b = inverse_b (R_b - sum over earlier blocks of (diag(b) A)_bj X_j), as products of two-term operands. The ten
  // 16 x 16 matrices are laid out as A fragments in the place of the decays, tokens in the order of token_of; a warp takes
  // 16 columns.
  uint4* matrices = reinterpret_cast<uint4*>(gs);  // block (b, j) at (b (b + 1) / 2 + j) * 64; (b, b) the inverse
  if (warp < 10) {
    const int b = warp < 1 ? 0 : warp < 3 ? 1 : warp < 6 ? 2 : 3, j = warp - b * (b + 1) / 2;
    float x[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const int row = b * kBlock + g + ((e >> 1) & 1) * 8, col = j * kBlock + token_of(c, e);
      x[e] = b != j ? -at[col * kPitchA + row] : row == col ? 1.0f : row > col ? at[row * kPitchA + col] : 0.0f;
    }
    store_fragment(matrices + warp * 64 + lane, x);
  }
  auto solve = [&](float* column, float4* result) {
    uint32_t xh[3][2][2], xl[3][2][2];  // blocks solved so far, as B operands of two tiles of eight columns
    auto swap_layout = [&](int b, const float (&acc)[2][4], uint32_t (&h)[2][2], uint32_t (&l)[2][2]) {
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        float* to = column + (b * kBlock + g) * pitch + n * 8 + 2 * c;
        *reinterpret_cast<float2*>(to) = make_float2(acc[n][0], acc[n][1]);
        *reinterpret_cast<float2*>(to + 8 * pitch) = make_float2(acc[n][2], acc[n][3]);
      }
      __syncwarp();
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        const float* from = column + (b * kBlock + c) * pitch + n * 8 + g;
        split_pair(from[0], from[4 * pitch], h[n][0], l[n][0]);
        split_pair(from[8 * pitch], from[12 * pitch], h[n][1], l[n][1]);
      }
      __syncwarp();
    };
    auto product = [&](int at_matrix, const uint32_t (&h)[2][2], const uint32_t (&l)[2][2], float (&acc)[2][4]) {
      const uint4 ah = matrices[at_matrix * 64 + lane], al = matrices[at_matrix * 64 + 32 + lane];
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        mma_bf16_16816(acc[n], ah.x, ah.y, ah.z, ah.w, h[n][0], h[n][1]);
        mma_bf16_16816(acc[n], ah.x, ah.y, ah.z, ah.w, l[n][0], l[n][1]);
        mma_bf16_16816(acc[n], al.x, al.y, al.z, al.w, h[n][0], h[n][1]);
      }
    };
#pragma unroll
    for (int b = 0; b < kChunk / kBlock; ++b) {
      float acc[2][4];
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        const float* from = column + (b * kBlock + g) * pitch + n * 8 + 2 * c;
        const float2 lo = *reinterpret_cast<const float2*>(from), hi = *reinterpret_cast<const float2*>(from + 8 * pitch);
        acc[n][0] = lo.x;
        acc[n][1] = lo.y;
        acc[n][2] = hi.x;
        acc[n][3] = hi.y;
      }
#pragma unroll
      for (int j = 0; j < b; ++j) product(b * (b + 1) / 2 + j, xh[j], xl[j], acc);
      uint32_t rh[2][2], rl[2][2];
      swap_layout(b, acc, rh, rl);
#pragma unroll
      for (int n = 0; n < 2; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.0f;
      product(b * (b + 1) / 2 + b, rh, rl, acc);
      if (result) {
#pragma unroll
        for (int n = 0; n < 2; ++n)
          result[(size_t(b) * (o.vdim_pad / 8) + n) * 32 + lane] = make_float4(acc[n][0], acc[n][1], acc[n][2], acc[n][3]);
      }
      if (b < 3) {
        swap_layout(b, acc, xh[b < 3 ? b : 0], xl[b < 3 ? b : 0]);
      } else if (!result) {
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          float* to = column + (b * kBlock + g) * pitch + n * 8 + 2 * c;
          *reinterpret_cast<float2*>(to) = make_float2(acc[n][0], acc[n][1]);
          *reinterpret_cast<float2*>(to + 8 * pitch) = make_float2(acc[n][2], acc[n][3]);
        }
      }
    }
  };
  for (int v0 = 0; v0 < o.vdim_pad; v0 += dim) {
    const int width = min(dim, o.vdim_pad - v0), width_quads = width / 4;
    auto put_value = [&](int i, uint2 raw) {
      const int t = i / width_quads, d = (i - t * width_quads) * 4;
      const float b = beta[t];
      *reinterpret_cast<float4*>(ks + t * pitch + d) = make_float4(bf16_lo(raw.x) * b, bf16_hi(raw.x) * b, bf16_lo(raw.y) * b, bf16_hi(raw.y) * b);
    };
    auto fetch_value = [&](int i) {
      const int t = i / width_quads, d = (i - t * width_quads) * 4;
      return t < live ? *reinterpret_cast<const uint2*>(values + size_t(t) * p.channels + v0 + d) : make_uint2(0, 0);
    };
    int i = threadIdx.x;
    if (v0 == 0) {
#pragma unroll
      for (int n = 0; n < kValueQuads; ++n, i += kPrepareThreads)
        if (i < kChunk * width_quads) put_value(i, ahead[n]);
    }
    for (; i < kChunk * width_quads; i += kPrepareThreads) put_value(i, fetch_value(i));
    __syncthreads();
    const int unsolved = v0 == 0 ? dim : 0;  // columns of W still to come, ahead of the value columns
    for (int begin = warp * 16; begin < unsolved + width; begin += kWarps * 16) {
      const int value = begin - unsolved;
      if (value < 0)
        solve(qs + begin, nullptr);
      else
        solve(ks + value, v_out + size_t(v0 + value) / 8 * 32);
    }
    __syncthreads();
  }
  uint4* w_out = reinterpret_cast<uint4*>(own + layout.w);
  for (int tile = warp; tile < 4 * steps; tile += kWarps) {
    const int mt = tile / steps, kk = tile - mt * steps;
    const float* x = qs + (mt * 16 + g) * pitch + kk * 16 + 4 * c;
    store_fragment(w_out + size_t(tile) * 64 + lane, quad_at(x), quad_at(x + 8 * pitch));
  }
}

// Block (head, kColumns values), eight warps, the chunks one after the other. Warps 0-3 hold 16 rows each of U, warps 4-7
// of the output; every warp holds kTiles tiles of 16 key channels of the state. Operands are requested a phase ahead of
// their use.
constexpr int kThreads = 256;
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
  // Accumulator rows into the two terms of an operand; tokens in the order of token_of, key channels of a tile in the order
  // of store_fragment's quads.
  const int token_rows[2] = {token_place(g), token_place(g + 8)};
  const int channel_rows[2] = {(g >> 2) * 2 + (g & 1) + ((g >> 1) & 1) * 8, ((g >> 2) + 2) * 2 + (g & 1) + ((g >> 1) & 1) * 8};
  auto publish = [&](const float (&x)[kN][4], int row, const int (&places)[2], bf16* leading, bf16* rest) {
#pragma unroll
    for (int n = 0; n < kN; ++n) {
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t hi, lo;
        split_pair(x[n][2 * half], x[n][2 * half + 1], hi, lo);
        const int at = (row + places[half]) * kPitch + n * 8 + 2 * c;
        *reinterpret_cast<uint32_t*>(leading + at) = hi;
        *reinterpret_cast<uint32_t*>(rest + at) = lo;
      }
    }
  };
#pragma unroll
  for (int m = 0; m < kTiles; ++m)
    if (warp + 8 * m < steps) publish(s[m], (warp + 8 * m) * 16, channel_rows, state_leading, state_rest);
  __syncthreads();

  // acc[0] += A leading x B leading, acc[1] += A rest x B leading, acc[2] += A leading x B rest: three short chains instead
  // of a long one. A: a two-term fragment, B: two-term rows of `leading` / `rest` at `row`, this lane's row of the 16.
  auto multiply = [&](float (&acc)[3][kN][4], const uint4& ah, const uint4& al, const bf16* leading, const bf16* rest, int row) {
#pragma unroll
    for (int n = 0; n < kN; n += 2) {
      const int at = row * kPitch + (n + (matrix >> 1)) * 8;
      uint32_t b0, b1, b2, b3;
      ldmatrix_x4_trans(b0, b1, b2, b3, leading + at);
      mma_bf16_16816(acc[0][n], ah.x, ah.y, ah.z, ah.w, b0, b1);
      mma_bf16_16816(acc[0][n + 1], ah.x, ah.y, ah.z, ah.w, b2, b3);
      mma_bf16_16816(acc[1][n], al.x, al.y, al.z, al.w, b0, b1);
      mma_bf16_16816(acc[1][n + 1], al.x, al.y, al.z, al.w, b2, b3);
      ldmatrix_x4_trans(b0, b1, b2, b3, rest + at);
      mma_bf16_16816(acc[2][n], ah.x, ah.y, ah.z, ah.w, b0, b1);
      mma_bf16_16816(acc[2][n + 1], ah.x, ah.y, ah.z, ah.w, b2, b3);
    }
  };
  auto clear = [](float (&acc)[3][kN][4]) {
#pragma unroll
    for (int term = 0; term < 3; ++term)
#pragma unroll
      for (int n = 0; n < kN; ++n) acc[term][n][0] = acc[term][n][1] = acc[term][n][2] = acc[term][n][3] = 0.0f;
  };
  auto total = [](const float (&acc)[3][kN][4], int n, int e) { return acc[0][n][e] + (acc[1][n][e] + acc[2][n][e]); };
  const int own_row = (matrix & 1) * 8 + in_matrix;
  constexpr int kAhead = 8;  // K steps of an operand requested at once
  const int row_tile = warp & 3;
  const unsigned char* own = p.chunks + size_t(head) * layout.total;
  const size_t chunk_bytes = size_t(o.heads) * layout.total;
  auto operand_of = [&](const unsigned char* at) {
    return reinterpret_cast<const uint4*>(at + (warp < 4 ? layout.w : layout.q)) + size_t(row_tile) * steps * 64 + lane;
  };
  uint4 ah[kAhead], al[kAhead];
  auto request = [&](const uint4* operand, int kk) {
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
      if (kk + i < steps) {
        ah[i] = operand[size_t(kk + i) * 64];
        al[i] = operand[size_t(kk + i) * 64 + 32];
      }
    }
  };
  request(operand_of(own), 0);
  for (int chunk = 0; chunk < chunks; ++chunk, own += chunk_bytes) {
    // Requested for the second phase: the keys of this warp's first tile, the decay, B or V'.
    const uint4* keys = reinterpret_cast<const uint4*>(own + layout.k) + lane;
    const float* decay = reinterpret_cast<const float*>(own + layout.decay);
    const uint4* inside = reinterpret_cast<const uint4*>(own + layout.b) + size_t(row_tile) * 4 * 64 + lane;
    uint4 kh[4], kl[4], bh[4], bl[4];
    float4 v[kN];
    float decay_lo = 1.0f, decay_hi = 1.0f;
    if (warp < steps) {
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        kh[kk] = keys[size_t(warp * 4 + kk) * 64];
        kl[kk] = keys[size_t(warp * 4 + kk) * 64 + 32];
      }
      decay_lo = decay[warp * 16 + g];
      decay_hi = decay[warp * 16 + g + 8];
    }
    if (warp < 4) {
      const float4* from = reinterpret_cast<const float4*>(own + layout.v) + (size_t(row_tile) * (o.vdim_pad / 8) + first_value / 8) * 32 + lane;
#pragma unroll
      for (int n = 0; n < kN; ++n) v[n] = n * 8 < live_columns ? from[n * 32] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    } else {
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        if (kk <= row_tile) {
          bh[kk] = inside[size_t(kk) * 64];
          bl[kk] = inside[size_t(kk) * 64 + 32];
        }
      }
    }
    float acc[3][kN][4];
    clear(acc);
    for (int kk = 0; kk < steps; kk += kAhead) {
      if (kk) request(operand_of(own), kk);
#pragma unroll
      for (int i = 0; i < kAhead; ++i)
        if (kk + i < steps) multiply(acc, ah[i], al[i], state_leading, state_rest, (kk + i) * 16 + own_row);
    }
    if (chunk + 1 < chunks) request(operand_of(own + chunk_bytes), 0);
    if (warp < 4) {
      float u[kN][4];
#pragma unroll
      for (int n = 0; n < kN; ++n) {
        u[n][0] = v[n].x - total(acc, n, 0);
        u[n][1] = v[n].y - total(acc, n, 1);
        u[n][2] = v[n].z - total(acc, n, 2);
        u[n][3] = v[n].w - total(acc, n, 3);
      }
      publish(u, row_tile * 16, token_rows, write_leading, write_rest);
    }
    __syncthreads();  // the writes are there, and every warp is done with the staged state
#pragma unroll
    for (int m = 0; m < kTiles; ++m) {
      const int tile = warp + 8 * m;
      if (tile >= steps) break;
      if (m) {
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
          kh[kk] = keys[size_t(tile * 4 + kk) * 64];
          kl[kk] = keys[size_t(tile * 4 + kk) * 64 + 32];
        }
        decay_lo = decay[tile * 16 + g];
        decay_hi = decay[tile * 16 + g + 8];
      }
      float added[3][kN][4];
      clear(added);
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) multiply(added, kh[kk], kl[kk], write_leading, write_rest, kk * 16 + own_row);
#pragma unroll
      for (int n = 0; n < kN; ++n) {
        s[m][n][0] = fmaf(decay_lo, s[m][n][0], total(added, n, 0));
        s[m][n][1] = fmaf(decay_lo, s[m][n][1], total(added, n, 1));
        s[m][n][2] = fmaf(decay_hi, s[m][n][2], total(added, n, 2));
        s[m][n][3] = fmaf(decay_hi, s[m][n][3], total(added, n, 3));
      }
      publish(s[m], tile * 16, channel_rows, state_leading, state_rest);
    }
    if (warp >= 4) {
#pragma unroll
      for (int kk = 0; kk < 4; ++kk)
        if (kk <= row_tile) multiply(acc, bh[kk], bl[kk], write_leading, write_rest, kk * 16 + own_row);
      const int row = chunk * kChunk + row_tile * 16 + g;
      const size_t out_pitch = size_t(o.heads) * o.vdim_pad;
      float* out = o.out + size_t(row) * out_pitch + head * o.vdim_pad + first_value + 2 * c;
#pragma unroll
      for (int n = 0; n < kN; ++n) {
        if (n * 8 >= live_columns) continue;
        if (row < o.rows) *reinterpret_cast<float2*>(out + n * 8) = make_float2(total(acc, n, 0), total(acc, n, 1));
        if (row + 8 < o.rows) *reinterpret_cast<float2*>(out + 8 * out_pitch + n * 8) = make_float2(total(acc, n, 2), total(acc, n, 3));
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
  launch(delta_chunk_kernel, dim3(chunks, unsigned(p.outer.heads)), dim3(kPrepareThreads), prepare_shared(p.outer.dim_pad), stream, pdl, p);
  // Narrow blocks where wide ones would leave most of the chip idle.
  const bool narrow = p.outer.heads * ((p.outer.vdim_pad + 31) / 32) * 3 < multiprocessors * 2;
  if (p.outer.dim_pad <= 128)
    return narrow ? launch_scan<16, 1>(p, stream, pdl) : launch_scan<32, 1>(p, stream, pdl);
  narrow ? launch_scan<16, 2>(p, stream, pdl) : launch_scan<32, 2>(p, stream, pdl);
}

}  // namespace ei
