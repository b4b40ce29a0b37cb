// A gated linear recurrence a channel (the recurrent block of Griffin; De et al., "Griffin: Mixing Gated Linear
// Recurrences with Local Attention for Efficient Language Models"): from the two raw branches of a product, y and x,
//
//   u_t = conv(x + x_bias)            a short causal convolution a channel, with a bias, no activation
//   r_t = sigmoid(R u_t + r_bias)     R, I: one square matrix a block of neighbouring channels
//   i_t = sigmoid(I u_t + i_bias)
//   log a_t = rate * r_t              rate = -c softplus(lam), one number a channel, at most 0
//   S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t
//   out_t = S_t * gelu_tanh(y_t + y_bias)
//
// all of it 32-bit (the products R u and I u too: with bfloat16 matrices u enters the tensor cores as a sum of three
// bfloat16 numbers, which is the 32-bit number).  A sequence keeps S [width] and the convolution's inputs of its last
// `taps` positions in a ring, [taps][width], position p at entry p % taps: a token reads the entries of the taps - 1
// positions before it and writes its own, which is none of those, so many blocks can read a sequence's ring while one of
// them writes it.
//
// Longer portions:   conv (u of every token)  ->  gates (a_t and b_t = sqrt(1 - a^2) i u of every token, and for every
//                    tile of 64 tokens of a sequence what it does to a state: S -> A S + B)  ->  scan (a block
//                    composes the tiles before its own, walks its 64 tokens and writes their results)
// Steps of one token a sequence: everything in ONE kernel.
#include "attention_mma.cuh"

namespace xrt {

constexpr int LR_TILE = 64;     // tokens of a sequence that one block scans
constexpr int LR_MAX_TAPS = 9;

// What every kernel of the file takes; pointers that a kernel does not use are null.
struct RecurrenceArgs {
  const float* p;            // [T, p_stride]: y raw at 0, x raw at x_offset
  int p_stride, x_offset;
  const float *y_bias, *x_bias, *conv_w, *conv_b;  // [width], [width], [width, taps], [width]
  const float *r_bias, *i_bias, *rate;             // [width]
  float *state, *ring;       // [slots, width], [slots, taps, width] (null with one tap)
  const int *cu_seqlens, *seq_slot, *seq_start;
  int n_seqs, width, taps, blocks;
  float* u;                  // [T, width]
  float2* ab;                // [T, width] (a, b)
  float2* tiles;             // [sequences, tiles, width] (A, B) of every tile
  float* init;               // [sequences, width] the state the step began with
  int n_tiles;
};

// The division and the root by the special-function unit (2^-22 and 2^-23 of the result).
__device__ __forceinline__ float lr_sigmoid(float z) { return __fdividef(1.0f, 1.0f + expf(-z)); }
__device__ __forceinline__ float lr_sqrt(float x) {
  float y;
  asm("sqrt.approx.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// (a, b) of a channel from its gates before their sigmoids (biases added) and its u.  With m = a - 1 (which keeps its
// digits where a is close to 1) 1 - a^2 = -m (2 + m).
__device__ __forceinline__ float2 lr_step_of(float r_raw, float i_raw, float u, float rate) {
  const float m = expm1f(rate * lr_sigmoid(r_raw));
  return make_float2(1.0f + m, lr_sqrt(-m * (2.0f + m)) * lr_sigmoid(i_raw) * u);
}

// The convolution's input of position `pos` (channel c): of this step's tokens where pos >= start, else of the ring.
__device__ __forceinline__ float lr_input(const RecurrenceArgs& a, int slot, int begin, int start, int pos, int c) {
  if (pos < 0) return 0.f;
  if (pos >= start) return a.p[(size_t)(begin + pos - start) * a.p_stride + a.x_offset + c] + a.x_bias[c];
  return a.ring[((size_t)slot * a.taps + pos % a.taps) * a.width + c];
}

// One thread a channel, 16 tokens of a sequence a block.
constexpr int LR_CONV_TOKENS = 16;
template <int TAPS>  // 0: any number up to LR_MAX_TAPS
__global__ void __launch_bounds__(128) lr_conv_kernel(const RecurrenceArgs a) {
  constexpr int MOST = TAPS > 0 ? TAPS : LR_MAX_TAPS;
  pdl_trigger();
  pdl_wait();
  const int s = blockIdx.z, slot = a.seq_slot[s];
  const int begin = a.cu_seqlens[s], len = a.cu_seqlens[s + 1] - begin;
  const int l0 = blockIdx.y * LR_CONV_TOKENS;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (slot < 0 || l0 >= len || c >= a.width) return;
  const int taps = TAPS > 0 ? TAPS : a.taps, start = a.seq_start[s];
  float w[MOST], in[MOST];  // in[j]: the input under tap j of the token that comes next
#pragma unroll
  for (int j = 0; j < MOST; ++j) {
    w[j] = j < taps ? a.conv_w[(size_t)c * taps + j] : 0.f;
    in[j] = j < taps - 1 ? lr_input(a, slot, begin, start, start + l0 - (taps - 1) + j, c) : 0.f;
  }
  const float bias = a.conv_b[c], xb = a.x_bias[c];
  const float* x = a.p + (size_t)(begin + l0) * a.p_stride + a.x_offset + c;
  float* u = a.u + (size_t)(begin + l0) * a.width + c;
  float next[LR_CONV_TOKENS];
#pragma unroll
  for (int l = 0; l < LR_CONV_TOKENS; ++l) next[l] = l0 + l < len ? x[(size_t)l * a.p_stride] + xb : 0.f;
#pragma unroll
  for (int l = 0; l < LR_CONV_TOKENS; ++l) {
    float acc = bias;
#pragma unroll
    for (int j = 0; j < MOST; ++j) {
      if (j == taps - 1) in[j] = next[l];
      if (j < taps) acc = fmaf(w[j], in[j], acc);
    }
    if (l0 + l < len) u[(size_t)l * a.width] = acc;
#pragma unroll
    for (int j = 0; j + 1 < MOST; ++j) in[j] = in[j + 1];
  }
}

// Folds 64 tokens' (a, b) of a block's channels, in shared memory [token][column], into (A, B) a column; 128 threads
// for at most 64 columns, two halves of the tokens side by side.
template <int LD>
__device__ __forceinline__ void lr_fold_tile(const float2 (*ab)[LD], int columns, float2* half, float2* out) {
  const int c = threadIdx.x & 63, part = threadIdx.x >> 6;
  float2 total = make_float2(1.f, 0.f);
#pragma unroll 8
  for (int l = part * 32; l < part * 32 + 32; ++l) {
    const float2 v = ab[l][c];
    total = make_float2(total.x * v.x, fmaf(total.y, v.x, v.y));
  }
  if (part == 1) half[c] = total;
  __syncthreads();
  if (part == 0 && c < columns) out[c] = make_float2(total.x * half[c].x, fmaf(total.y, half[c].x, half[c].y));
}

// Gates from the two products made elsewhere (any matrix size, 32-bit matrices): r_raw, i_raw [T, width].
__global__ void __launch_bounds__(128)
lr_gates_kernel(const RecurrenceArgs a, const float* __restrict__ r_raw, const float* __restrict__ i_raw) {
  pdl_trigger();
  pdl_wait(r_raw, i_raw);
  const int s = blockIdx.z, tile = blockIdx.y, slot = a.seq_slot[s];
  const int begin = a.cu_seqlens[s], len = a.cu_seqlens[s + 1] - begin;
  const int l0 = tile * LR_TILE, c = blockIdx.x * blockDim.x + threadIdx.x;
  if (slot < 0 || l0 >= len || c >= a.width) return;
  if (tile == 0) a.init[(size_t)s * a.width + c] = a.state[(size_t)slot * a.width + c];
  const float rate = a.rate[c], rb = a.r_bias[c], ib = a.i_bias[c];
  float2 total = make_float2(1.f, 0.f);
  const int n = min(LR_TILE, len - l0);
  for (int l = 0; l < n; ++l) {
    const size_t e = (size_t)(begin + l0 + l) * a.width + c;
    const float2 v = lr_step_of(r_raw[e] + rb, i_raw[e] + ib, a.u[e], rate);
    a.ab[e] = v;
    total = make_float2(total.x * v.x, fmaf(total.y, v.x, v.y));
  }
  a.tiles[((size_t)s * a.n_tiles + tile) * a.width + c] = total;
}

// x = hi + mid + lo exactly (three bfloat16 numbers hold the 24 bits of a 32-bit one); pairs of neighbours packed.
__device__ __forceinline__ void lr_split3(float2 x, uint32_t& hi, uint32_t& mid, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x.x, x.y);
  const float2 hf = __bfloat1622float2(h);
  x.x -= hf.x;
  x.y -= hf.y;
  const __nv_bfloat162 m = __floats2bfloat162_rn(x.x, x.y);
  const float2 mf = __bfloat1622float2(m);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x.x - mf.x, x.y - mf.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  mid = *reinterpret_cast<const uint32_t*>(&m);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}

// Gates on the tensor cores: a block has 64 tokens of a sequence and 64 channels of one block of channels, and both
// matrices; stretches of 32 inputs at a time, double-buffered.  size = width / blocks, a multiple of 8.
constexpr int LR_K = 32, LR_LD = LR_K + 8;
struct LrGateTiles {
  float u[2][LR_TILE][LR_LD];
  __nv_bfloat16 w[2][2][64][LR_LD];
};
__global__ void __launch_bounds__(128)
lr_gates_mma_kernel(const RecurrenceArgs a, const __nv_bfloat16* __restrict__ w_r, const __nv_bfloat16* __restrict__ w_i,
                    int size, int out_tiles) {
  __shared__ __align__(16) union {
    LrGateTiles in;
    float2 ab[LR_TILE][66];
  } sh;
  __shared__ float2 half[64];
  pdl_trigger();
  pdl_wait(w_r, w_i);
  const int s = blockIdx.z, tile = blockIdx.y, slot = a.seq_slot[s];
  const int begin = a.cu_seqlens[s], len = a.cu_seqlens[s + 1] - begin;
  const int l0 = tile * LR_TILE;
  if (slot < 0 || l0 >= len) return;
  const int block = blockIdx.x / out_tiles, o0 = (blockIdx.x - block * out_tiles) * 64;
  const int n_rows = min(LR_TILE, len - l0), n_out = min(64, size - o0);
  const float* u_rows = a.u + (size_t)(begin + l0) * a.width + (size_t)block * size;
  const __nv_bfloat16* wr = w_r + ((size_t)block * size + o0) * size;
  const __nv_bfloat16* wi = w_i + ((size_t)block * size + o0) * size;
  auto fetch = [&](int k0, int buffer) {
    for (int e = threadIdx.x; e < LR_TILE * (LR_K / 4); e += 128) {
      const int r = e / (LR_K / 4), c = (e % (LR_K / 4)) * 4;
      const bool live = r < n_rows && k0 + c < size;
      cp_async_16(smem_addr(&sh.in.u[buffer][r][c]), live ? u_rows + (size_t)r * a.width + k0 + c : a.u, live ? 16 : 0);
    }
    for (int e = threadIdx.x; e < 2 * 64 * (LR_K / 8); e += 128) {
      const int which = e / (64 * (LR_K / 8)), rest = e % (64 * (LR_K / 8)), r = rest / (LR_K / 8), c = (rest % (LR_K / 8)) * 8;
      const bool live = r < n_out && k0 + c < size;
      const __nv_bfloat16* from = which ? wi : wr;
      cp_async_16(smem_addr(&sh.in.w[buffer][which][r][c]), live ? from + (size_t)r * size + k0 + c : w_r, live ? 16 : 0);
    }
    cp_async_commit();
  };
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int row = warp * 16 + g;
  float acc[2][8][4];
#pragma unroll
  for (int which = 0; which < 2; ++which)
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[which][j][e] = 0.f;
  const int steps = (size + LR_K - 1) / LR_K;
  fetch(0, 0);
  for (int i = 0; i < steps; ++i) {
    const int b = i & 1;
    if (i + 1 < steps) { fetch((i + 1) * LR_K, b ^ 1); cp_async_wait<1>(); }
    else cp_async_wait<0>();
    __syncthreads();
#pragma unroll
    for (int ks = 0; ks < LR_K; ks += 16) {
      uint32_t part[3][4];
#pragma unroll
      for (int e = 0; e < 4; ++e)
        lr_split3(*reinterpret_cast<const float2*>(&sh.in.u[b][row + (e & 1) * 8][ks + (e >> 1) * 8 + 2 * t]), part[0][e],
                  part[1][e], part[2][e]);
#pragma unroll
      for (int which = 0; which < 2; ++which)
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const __nv_bfloat16* wp = &sh.in.w[b][which][j * 8 + g][ks + 2 * t];
          const uint32_t b0 = *reinterpret_cast<const uint32_t*>(wp), b1 = *reinterpret_cast<const uint32_t*>(wp + 8);
          mma_16816(acc[which][j], part[2], b0, b1);  // the small terms first
          mma_16816(acc[which][j], part[1], b0, b1);
          mma_16816(acc[which][j], part[0], b0, b1);
        }
    }
    __syncthreads();
  }
  // the steps of this block's tokens and channels; rows beyond the sequence leave a state as it is
  const int c0 = block * size + o0;
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int col = j * 8 + 2 * t;
    if (col < n_out) {  // sizes are multiples of 8: both columns or none
      const int c = c0 + col;
      const float2 rb = *reinterpret_cast<const float2*>(a.r_bias + c), ib = *reinterpret_cast<const float2*>(a.i_bias + c);
      const float2 rate = *reinterpret_cast<const float2*>(a.rate + c);
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int r = row + h * 8;
        float4 v = make_float4(1.f, 0.f, 1.f, 0.f);
        if (r < n_rows) {
          const size_t e = (size_t)(begin + l0 + r) * a.width + c;
          const float2 u = *reinterpret_cast<const float2*>(a.u + e);
          const float2 v0 = lr_step_of(acc[0][j][2 * h] + rb.x, acc[1][j][2 * h] + ib.x, u.x, rate.x);
          const float2 v1 = lr_step_of(acc[0][j][2 * h + 1] + rb.y, acc[1][j][2 * h + 1] + ib.y, u.y, rate.y);
          v = make_float4(v0.x, v0.y, v1.x, v1.y);
          *reinterpret_cast<float4*>(a.ab + e) = v;
        }
        *reinterpret_cast<float4*>(&sh.ab[r][col]) = v;
      }
    }
  }
  __syncthreads();
  if (tile == 0 && threadIdx.x < n_out)
    a.init[(size_t)s * a.width + c0 + threadIdx.x] = a.state[(size_t)slot * a.width + c0 + threadIdx.x];
  lr_fold_tile<66>(sh.ab, n_out, half, a.tiles + ((size_t)s * a.n_tiles + tile) * a.width + c0);
}

// One thread a channel, one tile of tokens a block.  Every block takes the state at its tile's start from what the tiles
// before it do to the step's first state, in order.  The last tile's block leaves the sequence's state and ring.
template <typename TO>
__global__ void __launch_bounds__(128, 4) lr_scan_kernel(TO* __restrict__ out, const RecurrenceArgs a) {
  pdl_trigger();
  pdl_wait();
  const int s = blockIdx.z, tile = gridDim.y - 1 - blockIdx.y, slot = a.seq_slot[s];  // later tiles have more before them
  const int begin = a.cu_seqlens[s], len = a.cu_seqlens[s + 1] - begin;
  const int l0 = tile * LR_TILE, c = blockIdx.x * blockDim.x + threadIdx.x;
  if (slot < 0 || l0 >= len || c >= a.width) return;
  float state = a.init[(size_t)s * a.width + c];
  const float2* before = a.tiles + (size_t)s * a.n_tiles * a.width + c;
#pragma unroll 8
  for (int i = 0; i < tile; ++i) {
    const float2 v = before[(size_t)i * a.width];
    state = fmaf(v.x, state, v.y);
  }
  const float yb = a.y_bias[c];
  const int n = min(LR_TILE, len - l0);
  const size_t first = (size_t)(begin + l0);
  const float2* ab = a.ab + first * a.width + c;
  const float* y = a.p + first * a.p_stride + c;
  TO* o = out + first * a.width + c;
  // several tokens' loads in flight: a load may not pass a store that could alias it, so they are all asked for before
  // the first result is written
  constexpr int AHEAD = 16;
  for (int at = 0; at < n; at += AHEAD) {
    float2 v[AHEAD];
    float g[AHEAD];
#pragma unroll
    for (int j = 0; j < AHEAD; ++j) {
      const bool live = at + j < n;
      v[j] = live ? ab[(size_t)(at + j) * a.width] : make_float2(1.f, 0.f);
      g[j] = live ? y[(size_t)(at + j) * a.p_stride] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < AHEAD; ++j) {
      state = fmaf(v[j].x, state, v[j].y);
      if (at + j < n) o[(size_t)(at + j) * a.width] = from_float<TO>(state * gelu_tanh_gate(g[j] + yb));
    }
  }
  if (l0 + n < len) return;
  a.state[(size_t)slot * a.width + c] = state;
  if (a.taps > 1) {
    const int start = a.seq_start[s];
    for (int l = max(0, len - a.taps); l < len; ++l)
      a.ring[((size_t)slot * a.taps + (start + l) % a.taps) * a.width + c] =
          a.p[(size_t)(begin + l) * a.p_stride + a.x_offset + c] + a.x_bias[c];
  }
}

// Steps of one token a sequence, bfloat16 matrices: a block has 32 channels of one block of channels (a warp 8) and
// both matrices' rows for them, and walks the step's rows 16 at a time.  The block's weights are asked for before the
// wait for the kernel before it.  Convolution inputs of the whole block of channels are worked out by every block that
// needs them (at most LR_STEP_K at a time, in shared memory), a thread a channel, several rows' loads in flight; what
// the end needs (states, gate inputs, biases) is asked for before the products.  Rows of no sequence (slot < 0) give
// zeros.  TAPS 0: any number up to LR_MAX_TAPS.
constexpr int LR_STEP_K = 256, LR_STEP_LD = LR_STEP_K + 4, LR_STEP_ROWS = 16, LR_STEP_GROUP = 4;
template <int TAPS>
__global__ void __launch_bounds__(128)
lr_step_kernel(__nv_bfloat16* __restrict__ out, const RecurrenceArgs a, const __nv_bfloat16* __restrict__ w_r,
               const __nv_bfloat16* __restrict__ w_i, const int* __restrict__ tok_slot, const int* __restrict__ tok_pos,
               int n_tokens, int size) {
  constexpr int MOST = TAPS > 0 ? TAPS : LR_MAX_TAPS;
  __shared__ __align__(16) float us[LR_STEP_ROWS][LR_STEP_LD];
  __shared__ int slots[LR_STEP_ROWS], places[LR_STEP_ROWS];
  __shared__ int entries[LR_STEP_ROWS][LR_MAX_TAPS];  // ring row of the input under each tap but the last (-1: before the start)
  pdl_trigger();
  const int block = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int taps = TAPS > 0 ? TAPS : a.taps;
  const int o_row = blockIdx.x * 32 + warp * 8;  // this warp's first channel inside the block of channels
  constexpr int PIECES = LR_STEP_K / 32;
  uint4 wr[PIECES], wi[PIECES];
  // lane (g, t) holds inputs 32 j + 8 t .. + 8 of channel g: the two products of a stretch of 32 inputs take four of
  // them each, so a lane's operands are neighbours (any order of k does, as long as both operands agree)
  auto load_weights = [&](int k0) {
    const size_t at = ((size_t)block * size + o_row + g) * size + k0 + 8 * t;
#pragma unroll
    for (int j = 0; j < PIECES; ++j) {
      const bool live = o_row + g < size && k0 + 32 * j + 8 * t < size;
      wr[j] = live ? __ldg(reinterpret_cast<const uint4*>(w_r + at + 32 * j)) : make_uint4(0u, 0u, 0u, 0u);
      wi[j] = live ? __ldg(reinterpret_cast<const uint4*>(w_i + at + 32 * j)) : make_uint4(0u, 0u, 0u, 0u);
    }
  };
  load_weights(0);
  // the step's arrays were written before the step began, weights long before
  const int o = o_row + 2 * t, c_own = block * size + o;  // this lane's two channels (sizes are multiples of 8)
  const bool own = o < size;
  float2 rb = make_float2(0.f, 0.f), ib = rb, yb = rb, xb = rb, rate = rb;
  if (own) {
    rb = *reinterpret_cast<const float2*>(a.r_bias + c_own); ib = *reinterpret_cast<const float2*>(a.i_bias + c_own);
    yb = *reinterpret_cast<const float2*>(a.y_bias + c_own); xb = *reinterpret_cast<const float2*>(a.x_bias + c_own);
    rate = *reinterpret_cast<const float2*>(a.rate + c_own);
  }
  const bool one_stretch = size <= LR_STEP_K;
  bool waited = false;
  for (int row0 = 0; row0 < n_tokens; row0 += LR_STEP_ROWS) {
    const int n_rows = min(LR_STEP_ROWS, n_tokens - row0);
    __syncthreads();
    if (threadIdx.x < LR_STEP_ROWS) {
      const int r = threadIdx.x;
      const int slot = r < n_rows ? tok_slot[row0 + r] : -1, pos = r < n_rows ? tok_pos[row0 + r] : 0;
      slots[r] = slot;
      places[r] = pos;
      for (int j = 0; j + 1 < taps; ++j) {
        const int p = pos - (taps - 1) + j;
        entries[r][j] = p >= 0 && slot >= 0 ? slot * taps + p % taps : -1;
      }
    }
    __syncthreads();
    if (!waited) { pdl_wait(w_r, w_i, tok_slot, tok_pos); waited = true; }
    // u of rows r0 .. r0 + LR_STEP_GROUP and channel c of all channels
    auto conv = [&](int r0, int c, float (&u)[LR_STEP_GROUP]) {
      float in[LR_STEP_GROUP][MOST];
      const float bias = a.x_bias[c];
#pragma unroll
      for (int i = 0; i < LR_STEP_GROUP; ++i) {
        const bool live = slots[r0 + i] >= 0;
#pragma unroll
        for (int j = 0; j < MOST; ++j) {
          in[i][j] = 0.f;
          if (j == taps - 1) {
            if (live) in[i][j] = a.p[(size_t)(row0 + r0 + i) * a.p_stride + a.x_offset + c] + bias;
          } else if (j < taps - 1 && live) {
            const int e = entries[r0 + i][j];
            if (e >= 0) in[i][j] = a.ring[(size_t)e * a.width + c];
          }
        }
      }
      const float cb = a.conv_b[c];
#pragma unroll
      for (int i = 0; i < LR_STEP_GROUP; ++i) u[i] = cb;
#pragma unroll
      for (int j = 0; j < MOST; ++j) {
        if (j < taps) {
          const float w = a.conv_w[(size_t)c * taps + j];
#pragma unroll
          for (int i = 0; i < LR_STEP_GROUP; ++i) u[i] = fmaf(w, in[i][j], u[i]);
        }
      }
    };
    // this lane's states and branches, rows g and g + 8
    float2 st[2], yv[2], xv[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int r = g + 8 * h;
      st[h] = yv[h] = xv[h] = make_float2(0.f, 0.f);
      if (own && slots[r] >= 0) {
        const float* row = a.p + (size_t)(row0 + r) * a.p_stride;
        st[h] = make_float2(a.state[(size_t)slots[r] * a.width + c_own], a.state[(size_t)slots[r] * a.width + c_own + 1]);
        yv[h] = make_float2(row[c_own], row[c_own + 1]);
        xv[h] = make_float2(row[a.x_offset + c_own], row[a.x_offset + c_own + 1]);
      }
    }
    float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    float2 u_own[2] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
    for (int k0 = 0; k0 < size; k0 += LR_STEP_K) {
      const int stretch = min(LR_STEP_K, (size - k0 + 31) / 32 * 32);
      if (k0 > 0) __syncthreads();
      for (int k = threadIdx.x; k < stretch; k += 128) {
#pragma unroll
        for (int r0 = 0; r0 < LR_STEP_ROWS; r0 += LR_STEP_GROUP) {
          float u[LR_STEP_GROUP] = {0.f, 0.f, 0.f, 0.f};
          if (r0 < n_rows && k0 + k < size) conv(r0, block * size + k0 + k, u);
#pragma unroll
          for (int i = 0; i < LR_STEP_GROUP; ++i) us[r0 + i][k] = u[i];
        }
      }
      if (!one_stretch) load_weights(k0);
      __syncthreads();
      if (own && o >= k0 && o < k0 + LR_STEP_K) {  // two neighbours of one stretch: the stretch is even
#pragma unroll
        for (int h = 0; h < 2; ++h) u_own[h] = make_float2(us[g + 8 * h][o - k0], us[g + 8 * h][o - k0 + 1]);
      }
#pragma unroll
      for (int j = 0; j < PIECES; ++j) {
        if (32 * j < stretch) {
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const float4 lo_row = *reinterpret_cast<const float4*>(&us[g][32 * j + 8 * t + 4 * half]);
            const float4 hi_row = *reinterpret_cast<const float4*>(&us[g + 8][32 * j + 8 * t + 4 * half]);
            uint32_t part[3][4];
            lr_split3(make_float2(lo_row.x, lo_row.y), part[0][0], part[1][0], part[2][0]);
            lr_split3(make_float2(hi_row.x, hi_row.y), part[0][1], part[1][1], part[2][1]);
            lr_split3(make_float2(lo_row.z, lo_row.w), part[0][2], part[1][2], part[2][2]);
            lr_split3(make_float2(hi_row.z, hi_row.w), part[0][3], part[1][3], part[2][3]);
            const uint32_t r0 = half ? wr[j].z : wr[j].x, r1 = half ? wr[j].w : wr[j].y;
            const uint32_t i0 = half ? wi[j].z : wi[j].x, i1 = half ? wi[j].w : wi[j].y;
#pragma unroll
            for (int term = 2; term >= 0; --term) {
              mma_16816(acc[0], part[term], r0, r1);
              mma_16816(acc[1], part[term], i0, i1);
            }
          }
        }
      }
    }
    if (!own) continue;
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int r = g + 8 * h, slot = slots[r];
      if (r >= n_rows) continue;
      __nv_bfloat162* dst = reinterpret_cast<__nv_bfloat162*>(out + (size_t)(row0 + r) * a.width + c_own);
      if (slot < 0) {
        *dst = __floats2bfloat162_rn(0.f, 0.f);
        continue;
      }
      const float2 v0 = lr_step_of(acc[0][2 * h] + rb.x, acc[1][2 * h] + ib.x, u_own[h].x, rate.x);
      const float2 v1 = lr_step_of(acc[0][2 * h + 1] + rb.y, acc[1][2 * h + 1] + ib.y, u_own[h].y, rate.y);
      const float2 s = make_float2(fmaf(v0.x, st[h].x, v0.y), fmaf(v1.x, st[h].y, v1.y));
      float* state = a.state + (size_t)slot * a.width + c_own;
      state[0] = s.x;
      state[1] = s.y;
      if (taps > 1) {
        float* ring = a.ring + ((size_t)slot * taps + places[r] % taps) * a.width + c_own;
        ring[0] = xv[h].x + xb.x;
        ring[1] = xv[h].y + xb.y;
      }
      *dst = __floats2bfloat162_rn(s.x * gelu_tanh_gate(yv[h].x + yb.x), s.y * gelu_tanh_gate(yv[h].y + yb.y));
    }
  }
}

}  // namespace xrt

// u [T, width] of the step's tokens (rows of no sequence are not written).
XRT_EXPORT int xrt_recurrence_conv(const xrt::RecurrenceArgs* args, int max_new, cudaStream_t stream) {
  const xrt::RecurrenceArgs& a = *args;
  if (a.n_seqs < 0 || a.width <= 0 || a.taps < 1 || max_new < 0 || (a.taps > 1 && a.ring == nullptr)) return XRT_ERR_ARGUMENT;
  if (a.taps > xrt::LR_MAX_TAPS || a.n_seqs > 65535) return XRT_ERR_UNSUPPORTED;
  if (a.n_seqs == 0 || max_new == 0) return XRT_OK;
  const dim3 grid((a.width + 127) / 128, (max_new + xrt::LR_CONV_TOKENS - 1) / xrt::LR_CONV_TOKENS, a.n_seqs);
  if (grid.y > 65535) return XRT_ERR_UNSUPPORTED;
#define XRT_LR_CONV(TAPS) xrt::launch_kernel(xrt::lr_conv_kernel<TAPS>, grid, dim3(128), 0, stream, a)
  switch (a.taps) {
    case 2: XRT_LR_CONV(2); break;
    case 3: XRT_LR_CONV(3); break;
    case 4: XRT_LR_CONV(4); break;
    default: XRT_LR_CONV(0);
  }
#undef XRT_LR_CONV
  return xrt::launch_status();
}

// (a, b) of every token and what every tile of 64 tokens does to a state.  w_r, w_i: bfloat16 [blocks, size, size] with
// a size that is a multiple of 8 (16-byte aligned), or null: then r_raw, i_raw float32 [T, width] hold the products.
XRT_EXPORT int xrt_recurrence_gates(const xrt::RecurrenceArgs* args, const void* w_r, const void* w_i, const float* r_raw,
                                    const float* i_raw, int max_new, cudaStream_t stream) {
  const xrt::RecurrenceArgs& a = *args;
  if (a.n_seqs < 0 || a.width <= 0 || a.blocks <= 0 || a.width % a.blocks || max_new < 0 ||
      a.n_tiles < (max_new + xrt::LR_TILE - 1) / xrt::LR_TILE)
    return XRT_ERR_ARGUMENT;
  if (a.n_seqs > 65535 || a.n_tiles > 65535) return XRT_ERR_UNSUPPORTED;
  if (a.n_seqs == 0 || max_new == 0) return XRT_OK;
  const int size = a.width / a.blocks;
  if (w_r == nullptr || w_i == nullptr) {
    if (r_raw == nullptr || i_raw == nullptr) return XRT_ERR_ARGUMENT;
    xrt::launch_kernel(xrt::lr_gates_kernel, dim3((a.width + 127) / 128, a.n_tiles, a.n_seqs), dim3(128), 0, stream, a, r_raw,
                       i_raw);
    return xrt::launch_status();
  }
  if (size % 8 || (((uintptr_t)w_r | (uintptr_t)w_i | (uintptr_t)a.u | (uintptr_t)a.ab) & 15) ||
      (((uintptr_t)a.r_bias | (uintptr_t)a.i_bias | (uintptr_t)a.rate) & 7))
    return XRT_ERR_UNSUPPORTED;
  const int out_tiles = (size + 63) / 64;
  xrt::launch_kernel(xrt::lr_gates_mma_kernel, dim3(a.blocks * out_tiles, a.n_tiles, a.n_seqs), dim3(128), 0, stream, a,
                     (const __nv_bfloat16*)w_r, (const __nv_bfloat16*)w_i, size, out_tiles);
  return xrt::launch_status();
}

// out [T, width] in out_dtype; leaves the sequences' states and rings.
XRT_EXPORT int xrt_recurrence_scan(void* out, const xrt::RecurrenceArgs* args, int max_new, int out_dtype,
                                   cudaStream_t stream) {
  const xrt::RecurrenceArgs& a = *args;
  if (a.n_seqs < 0 || a.width <= 0 || max_new < 0 || a.n_tiles < (max_new + xrt::LR_TILE - 1) / xrt::LR_TILE)
    return XRT_ERR_ARGUMENT;
  if (a.n_seqs > 65535 || a.n_tiles > 65535) return XRT_ERR_UNSUPPORTED;
  if (a.n_seqs == 0 || max_new == 0) return XRT_OK;
  XRT_DISPATCH_DTYPE(out_dtype, TO, {
    xrt::launch_kernel(xrt::lr_scan_kernel<TO>, dim3((a.width + 127) / 128, a.n_tiles, a.n_seqs), dim3(128), 0, stream,
                       (TO*)out, a);
  });
  return xrt::launch_status();
}

// A step of one token a sequence in one launch: out bfloat16 [T, width]; w_r, w_i as for xrt_recurrence_gates.
XRT_EXPORT int xrt_recurrence_step(void* out, const xrt::RecurrenceArgs* args, const void* w_r, const void* w_i,
                                   const int* tok_slot, const int* tok_pos, int n_tokens, cudaStream_t stream) {
  const xrt::RecurrenceArgs& a = *args;
  if (n_tokens < 0 || a.width <= 0 || a.blocks <= 0 || a.width % a.blocks || a.taps < 1 || (a.taps > 1 && a.ring == nullptr))
    return XRT_ERR_ARGUMENT;
  const int size = a.width / a.blocks;
  if (size % 8 || a.taps > xrt::LR_MAX_TAPS || a.blocks > 65535 || (((uintptr_t)w_r | (uintptr_t)w_i) & 15) ||
      (((uintptr_t)out | (uintptr_t)a.r_bias | (uintptr_t)a.i_bias | (uintptr_t)a.y_bias | (uintptr_t)a.x_bias | (uintptr_t)a.rate) & 7))
    return XRT_ERR_UNSUPPORTED;
  if (n_tokens == 0) return XRT_OK;
#define XRT_LR_STEP(TAPS)                                                                                          \
  xrt::launch_kernel(xrt::lr_step_kernel<TAPS>, dim3((size + 31) / 32, a.blocks), dim3(128), 0, stream,              \
                     (__nv_bfloat16*)out, a, (const __nv_bfloat16*)w_r, (const __nv_bfloat16*)w_i, tok_slot, tok_pos, \
                     n_tokens, size)
  switch (a.taps) {
    case 2: XRT_LR_STEP(2); break;
    case 3: XRT_LR_STEP(3); break;
    case 4: XRT_LR_STEP(4); break;
    default: XRT_LR_STEP(0);
  }
#undef XRT_LR_STEP
  return xrt::launch_status();
}
