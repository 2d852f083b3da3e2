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

// Sixteen warps. Of A and B, warp w takes four columns of a diagonal block and, up to the twelfth, a tile below the
// diagonal.
constexpr int kPrepareThreads = 512;
__global__ void __launch_bounds__(kPrepareThreads) delta_chunk_kernel(const DeltaPromptParams p) {
  extern __shared__ __align__(16) float chunk_smem[];
  const OuterStateParams& o = p.outer;
  const int dim = o.dim_pad, pitch = row_pitch(dim), steps = dim / 16;
  float* at = chunk_smem;                          // diag(b) A transposed: at[j][t], j < t
  float* gs = at + kChunk * kPitchA;               // [kChunk][pitch]: cumulative logarithms of the decays
  float* ks = gs + kChunk * pitch;                 // [kChunk][pitch]: unit k, then columns of W
  float* qs = ks + kChunk * pitch;                 // [kChunk][pitch]: scaled unit q, then columns of V'
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

  // A and B inside the diagonal blocks, directly. Warp w: block w >> 2; rows g and g + 8 of it against columns
  // 2 (w & 3), + 1, and row g + 8 against the columns eight further on.
  {
    const int base = (warp >> 2) * kBlock, column = base + (warp & 3) * 2;
    const int t = base + g;
    float ka[3][2], qa[3][2];  // [row g, early column | row g + 8, early column | row g + 8, late column]
#pragma unroll
    for (int n = 0; n < 3; ++n) ka[n][0] = ka[n][1] = qa[n][0] = qa[n][1] = 0.0f;
#pragma unroll 2
    for (int d = 4 * c; d < dim; d += 16) {
      const float4 gl = quad_at(gs + t * pitch + d), gh = quad_at(gs + (t + 8) * pitch + d);
      const float4 kl = quad_at(ks + t * pitch + d), kh = quad_at(ks + (t + 8) * pitch + d);
      const float4 ql = quad_at(qs + t * pitch + d), qh = quad_at(qs + (t + 8) * pitch + d);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float4 early_g = quad_at(gs + (column + e) * pitch + d), early_k = quad_at(ks + (column + e) * pitch + d);
        const float4 late_g = quad_at(gs + (column + e + 8) * pitch + d), late_k = quad_at(ks + (column + e + 8) * pitch + d);
        const float4 x = times(early_k, exp_below(gl, early_g)), y = times(early_k, exp_between(gh, early_g)), z = times(late_k, exp_below(gh, late_g));
        ka[0][e] = dot(kl, x, ka[0][e]);
        qa[0][e] = dot(ql, x, qa[0][e]);
        ka[1][e] = dot(kh, y, ka[1][e]);
        qa[1][e] = dot(qh, y, qa[1][e]);
        ka[2][e] = dot(kh, z, ka[2][e]);
        qa[2][e] = dot(qh, z, qa[2][e]);
      }
    }
#pragma unroll
    for (int n = 0; n < 3; ++n)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        ka[n][e] += __shfl_xor_sync(0xffffffffu, ka[n][e], 1);
        ka[n][e] += __shfl_xor_sync(0xffffffffu, ka[n][e], 2);
        qa[n][e] += __shfl_xor_sync(0xffffffffu, qa[n][e], 1);
        qa[n][e] += __shfl_xor_sync(0xffffffffu, qa[n][e], 2);
      }
    if (c < 2) {  // the four lanes of a row hold the same sums; lane c writes column + c
      const int e = c, early = column + e, late = early + 8;
      const float ka0 = e ? ka[0][1] : ka[0][0], ka1 = e ? ka[1][1] : ka[1][0], ka2 = e ? ka[2][1] : ka[2][0];
      const float qa0 = e ? qa[0][1] : qa[0][0], qa1 = e ? qa[1][1] : qa[1][0], qa2 = e ? qa[2][1] : qa[2][0];
      at[early * kPitchA + t] = early < t ? ka0 * beta[t] : 0.0f;
      bm[t * kPitchB + early] = early <= t ? qa0 : 0.0f;
      at[early * kPitchA + t + 8] = ka1 * beta[t + 8];
      bm[(t + 8) * kPitchB + early] = qa1;
      at[late * kPitchA + t + 8] = late < t + 8 ? ka2 * beta[t + 8] : 0.0f;
      bm[(t + 8) * kPitchB + late] = late <= t + 8 ? qa2 : 0.0f;
    } else if (c == 2) {
      for (int e = 0; e < 2; ++e) {
        at[(column + 8 + e) * kPitchA + t] = 0.0f;
        bm[t * kPitchB + column + 8 + e] = 0.0f;
      }
    }
  }
  // Below the diagonal: tiles of 16 rows x 8 columns, through the end of the block ahead of the rows.
  if (warp < 12) {
    const int block = warp < 2 ? 1 : warp < 6 ? 2 : 3, column = (warp - (block == 1 ? 0 : block == 2 ? 2 : 6)) * 8;
    const int t0 = block * kBlock;
    float ka[3][4], qa[3][4];  // a chain per product of terms
#pragma unroll
    for (int n = 0; n < 3; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) ka[n][e] = qa[n][e] = 0.0f;
#pragma unroll 2
    for (int d = 4 * c; d < dim; d += 16) {
      const float4 turn = quad_at(gs + (t0 - 1) * pitch + d);
      const float4 e_lo = exp_between(quad_at(gs + (t0 + g) * pitch + d), turn), e_hi = exp_between(quad_at(gs + (t0 + g + 8) * pitch + d), turn);
      uint32_t kh[4], kl[4], qh[4], ql[4], bh[2], bl[2];
      split_rows(times(quad_at(ks + (t0 + g) * pitch + d), e_lo), times(quad_at(ks + (t0 + g + 8) * pitch + d), e_hi), kh, kl);
      split_rows(times(quad_at(qs + (t0 + g) * pitch + d), e_lo), times(quad_at(qs + (t0 + g + 8) * pitch + d), e_hi), qh, ql);
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
      const int t = t0 + g + (e >> 1) * 8, j = column + 2 * c + (e & 1);
      at[j * kPitchA + t] = (ka[0][e] + (ka[1][e] + ka[2][e])) * beta[t];
      bm[t * kPitchB + j] = qa[0][e] + (qa[1][e] + qa[2][e]);
    }
  }
  __syncthreads();

  // Operands that need no solving: q e^G, k e^(G_end - G) transposed, B, and the chunk's decay.
  const float* last = gs + (kChunk - 1) * pitch;
  uint4* q_out = reinterpret_cast<uint4*>(own + layout.q);
  uint4* k_out = reinterpret_cast<uint4*>(own + layout.k);
  uint4* b_out = reinterpret_cast<uint4*>(own + layout.b);
#pragma unroll 2
  for (int tile = warp; tile < 4 * steps; tile += kWarps) {
    const int mt = tile / steps, kk = tile - mt * steps;
    const int row = (mt * 16 + g) * pitch + kk * 16 + 4 * c;
    store_fragment(q_out + size_t(mt * steps + kk) * 64 + lane, times(quad_at(qs + row), exp_of(quad_at(gs + row))),
                   times(quad_at(qs + row + 8 * pitch), exp_of(quad_at(gs + row + 8 * pitch))));
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
  __syncthreads();

  // The inverses of the four unit lower triangular diagonal blocks, one column per thread, into the blocks' places in bm
  // (B has been written out): inverse[i][j] at bm[(16 b + i) pitch + 16 b + j].
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
    for (int i = 0; i < kBlock; ++i) bm[(base + i) * kPitchB + base + j] = x[i];
  }
  // Solves (I + diag(b) A) X = right-hand side in place, 16 rows at a time. Lanes l and l + 16 share a column: lane
  // l + 16 h works on the rows 8 h .. 8 h + 7 of a block for the part below the diagonal blocks, and on every second row
  // for the product with the block's inverse.
  const int half = lane >> 4;
  auto solve = [&](float* column, bool live_column) {
#pragma unroll 1
    for (int b = 0; b < kChunk / kBlock; ++b) {
      float x[8];
      float* own_rows = column + (b * kBlock + half * 8) * pitch;
      if (live_column && b) {
#pragma unroll
        for (int i = 0; i < 8; ++i) x[i] = own_rows[i * pitch];
#pragma unroll 4
        for (int j = 0; j < b * kBlock; ++j) {
          const float known = column[j * pitch];
          const float* a = at + j * kPitchA + b * kBlock + half * 8;
          const float4 v = quad_at(a), w = quad_at(a + 4);
          x[0] = fmaf(-v.x, known, x[0]);
          x[1] = fmaf(-v.y, known, x[1]);
          x[2] = fmaf(-v.z, known, x[2]);
          x[3] = fmaf(-v.w, known, x[3]);
          x[4] = fmaf(-w.x, known, x[4]);
          x[5] = fmaf(-w.y, known, x[5]);
          x[6] = fmaf(-w.z, known, x[6]);
          x[7] = fmaf(-w.w, known, x[7]);
        }
#pragma unroll
        for (int i = 0; i < 8; ++i) own_rows[i * pitch] = x[i];
      }
      __syncwarp();
      float r[kBlock];
      if (live_column) {
#pragma unroll
        for (int i = 0; i < kBlock; ++i) r[i] = column[(b * kBlock + i) * pitch];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const float* t = bm + (b * kBlock + 2 * i + half) * kPitchB + b * kBlock;
          float sum = 0.0f;
#pragma unroll
          for (int j = 0; j < 2 * i + 2; ++j) sum = fmaf(t[j], r[j], sum);  // row 2 i has a zero at its end
          x[i] = sum;
        }
      }
      __syncwarp();
      if (live_column)
#pragma unroll
        for (int i = 0; i < 8; ++i) column[(b * kBlock + 2 * i + half) * pitch] = x[i];
      __syncwarp();
    }
  };
  // The columns of W in place of k, those of V' in place of q, `dim` value columns at a time.
  for (int v0 = 0; v0 < o.vdim_pad; v0 += dim) {
    const int width = min(dim, o.vdim_pad - v0), width_quads = width / 4;
    auto put_value = [&](int i, uint2 raw) {
      const int t = i / width_quads, d = (i - t * width_quads) * 4;
      const float b = beta[t];
      *reinterpret_cast<float4*>(qs + t * pitch + d) = make_float4(bf16_lo(raw.x) * b, bf16_hi(raw.x) * b, bf16_lo(raw.y) * b, bf16_hi(raw.y) * b);
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
    if (v0 == 0) {
#pragma unroll 4
      for (int n = threadIdx.x; n < kChunk * quads; n += kPrepareThreads) {
        const int t = n / quads, d = (n - t * quads) * 4;
        const float4 e = exp_of(quad_at(gs + t * pitch + d));
        const float b = beta[t];
        float4* k = reinterpret_cast<float4*>(ks + t * pitch + d);
        *k = times(*k, make_float4(e.x * b, e.y * b, e.z * b, e.w * b));
      }
    }
    __syncthreads();
    const int unsolved = v0 == 0 ? dim : 0;  // columns of W still to come, ahead of the value columns
    for (int begin = warp * 16; begin < unsolved + width; begin += kWarps * 16) {
      const int column = begin + (lane & 15);
      solve(column < unsolved ? ks + column : qs + column - unsolved, column < unsolved + width);
    }
    __syncthreads();
    // V' in the order of the accumulators: [row tile][column tile of 8][lane].
    for (int tile = warp; tile < 4 * (width / 8); tile += kWarps) {
      const int mt = tile / (width / 8), nt = tile - mt * (width / 8);
      const float* x = qs + (mt * 16 + g) * pitch + nt * 8 + 2 * c;
      v_out[(size_t(mt) * (o.vdim_pad / 8) + v0 / 8 + nt) * 32 + lane] = make_float4(x[0], x[1], x[8 * pitch], x[8 * pitch + 1]);
    }
    if (v0 + dim < o.vdim_pad) __syncthreads();
  }
  uint4* w_out = reinterpret_cast<uint4*>(own + layout.w);
  for (int tile = warp; tile < 4 * steps; tile += kWarps) {
    const int mt = tile / steps, kk = tile - mt * steps;
    const float* x = ks + (mt * 16 + g) * pitch + kk * 16 + 4 * c;
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
