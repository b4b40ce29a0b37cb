// Rotation tables, and the fused step between the q/k/v product and attention:
// optional per-head RMSNorm of q and k, rotation of q and k, q written for the attention kernel
// and k, v written into the cache blocks of each token's sequence.
//
// Formulas of the reference:
//   angle = pos * scale / base^(2i/rope_dim), in 32-bit   crates/xrt-kernels/src/cpu/rope.rs:59-68
//   h[i]      = x0 * cos - x1 * sin                        crates/xrt-kernels/src/cpu/rope.rs:19-35
//   h[i+half] = x0 * sin + x1 * cos      (x0 = h[i], x1 = h[i + half]; split-half pairing)
// The reference pairs (i, i + half) only.  `interleaved` pairs (2i, 2i + 1) instead, for position
// encodings that rotate neighbours; dims from 2 * rope_half on are left as they are either way.
//   head norm = RMSNorm over each head slice, one weight   crates/xrt-models/src/llama.rs:1025-1040
//   order     = projection, head norm, rotation, cache     crates/xrt-models/src/llama.rs:488-503
#include "common.cuh"

namespace xrt {

// cos_sin[t, i] = (cos, sin) of pos[t] * scale / freq[i]; freq is the divisor table base^(2i/rd).
__global__ void rope_table_kernel(float2* __restrict__ cos_sin, const int* __restrict__ pos,
                                  const float* __restrict__ freq, float scale, int n_tokens, int half) {
  pdl_trigger();
  pdl_wait(pos, freq);
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n_tokens * half) return;
  const int t = i / half, p = i - t * half;
  const float angle = __fdiv_rn(__fmul_rn((float)pos[t], scale), freq[p]);
  float s, c;
  sincosf(angle, &s, &c);
  cos_sin[i] = make_float2(c, s);
}

// cos_sin[t, i] = magnitude * (cos, sin) of pos[t] * freq[i]: a table of frequencies of any make (scaled,
// blended between two scalings) and one factor on both cos and sin.  The angle is one 32-bit product; with freq_lo
// (what the 32-bit frequency lost of its 64-bit value) the product's own rounding error and pos * freq_lo are kept as
// a second 32-bit term d, and cos(a + d) = cos a cos d - sin a sin d, sin(a + d) = sin a cos d + cos a sin d: a far
// position's angle is then as exact as a near one's.
__global__ void rotation_table_kernel(float2* __restrict__ cos_sin, const int* __restrict__ pos,
                                      const float* __restrict__ freq, const float* __restrict__ freq_lo, float magnitude,
                                      int n_tokens, int half) {
  pdl_trigger();
  pdl_wait(pos, freq, freq_lo);
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n_tokens * half) return;
  const int t = i / half, p = i - t * half;
  const float position = (float)pos[t];
  const float angle = __fmul_rn(position, freq[p]);
  float s, c;
  sincosf(angle, &s, &c);
  if (freq_lo != nullptr) {
    const float d = __fmaf_rn(position, freq_lo[p], __fmaf_rn(position, freq[p], -angle));
    float sd, cd;
    sincosf(d, &sd, &cd);
    const float c0 = c;
    c = __fmaf_rn(c0, cd, -s * sd);
    s = __fmaf_rn(s, cd, c0 * sd);
  }
  cos_sin[i] = make_float2(c * magnitude, s * magnitude);
}

// What a layer may ask for beside norm, rotation and the cache write (all optional, all 32-bit):
//   bias       one float a column of the q/k/v row (laid out as the row is), added first
//   unit_norm  q and k heads are divided by their root mean square, without a weight
//   norm_dim   the divisor of the heads' mean of squares where the heads are laid out wider than they are (0: head_dim)
//   v_keep     the values (after the bias) are also written here in 32-bit, [tokens, v_keep_stride]
//   v_first    the cached value is (1 - v_blend) v + v_blend v_first[token], v_first rows of v_first_stride floats
//   v_dim      the value size of a head in v_keep and v_first, which hold the heads at their true size whatever
//              size the layer's heads are laid out at (0: head_dim)
//   v_unit     every value head is divided by its root mean square over v_dim (eps of the layer, no weight) before
//              it is kept, blended or cached
//   whole_q, whole_k   > 0: the RMSNorm of q (of k) runs over the WHOLE projection, all heads of a token at once, with
//              one weight a column ([heads * head_dim], laid out as the heads are); the number is the divisor of the
//              mean of squares (the projection's true size, which is smaller than heads * head_dim where the heads
//              are laid out wider than they are).  Every warp adds up its token's row by itself, in one order.
struct HeadExtras {
  int whole_q = 0;
  int whole_k = 0;
  const float* bias = nullptr;
  int unit_norm = 0;
  int norm_dim = 0;
  float* v_keep = nullptr;
  int v_keep_stride = 0;
  const float* v_first = nullptr;
  int v_first_stride = 0;
  float v_blend = 0.f;
  int v_dim = 0;
  int v_unit = 0;
};

// One warp per (token, head) among [q heads | k heads | v heads].  MAX_PER_LANE * 32 >= head_dim.
template <typename TN, typename TQ, typename TC, int MAX_PER_LANE>
__global__ void qk_rope_kv_write_kernel(
    TQ* __restrict__ q_out, TC* __restrict__ k_pool, TC* __restrict__ v_pool,
    const float* __restrict__ qkv, int row_stride, int k_offset, int v_offset,
    const TN* __restrict__ q_norm_w, const TN* __restrict__ k_norm_w, float eps,
    const float2* __restrict__ cos_sin, int rope_half,
    const int* __restrict__ tok_slot, const int* __restrict__ tok_pos,
    const int* __restrict__ block_table, int max_blocks,
    int n_heads, int n_kv_heads, int head_dim, int write_kv, int interleaved, const QueryTemp temp, const HeadExtras ex) {
  extern __shared__ float staged[];  // [warps][head_dim]
  pdl_trigger();
  pdl_wait(qkv, q_norm_w, k_norm_w, cos_sin, tok_slot, tok_pos, block_table);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x;
  const int head_slot = blockIdx.y * (blockDim.x >> 5) + warp;
  const int n_slots = n_heads + (write_kv ? 2 * n_kv_heads : 0);
  if (head_slot >= n_slots) return;
  const int slot = tok_slot[t];
  const int pos = tok_pos[t];

  // which of q / k / v, and which head of it
  int kind, head;
  if (head_slot < n_heads) { kind = 0; head = head_slot; }
  else if (head_slot < n_heads + n_kv_heads) { kind = 1; head = head_slot - n_heads; }
  else { kind = 2; head = head_slot - n_heads - n_kv_heads; }

  if (slot < 0) {  // a padding row: q is zeroed, the cache is not touched
    if (kind == 0)
      for (int d = lane; d < head_dim; d += 32)
        q_out[(size_t)t * n_heads * head_dim + head * head_dim + d] = from_float<TQ>(0.f);
    return;
  }

  const int column = (kind == 0 ? 0 : (kind == 1 ? k_offset : v_offset)) + head * head_dim;
  const float* src = qkv + (size_t)t * row_stride + column;
  float v[MAX_PER_LANE];
  float sq = 0.f;
#pragma unroll
  for (int j = 0; j < MAX_PER_LANE; ++j) {
    const int d = lane + 32 * j;
    v[j] = d < head_dim ? src[d] : 0.f;
    if (ex.bias != nullptr && d < head_dim) v[j] += ex.bias[column + d];
    sq = fmaf(v[j], v[j], sq);
  }
  const TN* norm_w = kind == 0 ? q_norm_w : (kind == 1 ? k_norm_w : nullptr);
  const float norm_dim = (float)(ex.norm_dim > 0 ? ex.norm_dim : head_dim);
  const int whole = kind == 0 ? ex.whole_q : (kind == 1 ? ex.whole_k : 0);
  if (norm_w != nullptr && whole > 0) {
    const float* all = qkv + (size_t)t * row_stride + (kind == 0 ? 0 : k_offset);
    const int n_all = (kind == 0 ? n_heads : n_kv_heads) * head_dim;
    float total = 0.f;
    for (int c = lane; c < n_all; c += 32) {
      const float a = all[c] + (ex.bias != nullptr ? ex.bias[(kind == 0 ? 0 : k_offset) + c] : 0.f);
      total = fmaf(a, a, total);
    }
    const float inv = 1.0f / sqrtf(warp_sum(total) / (float)whole + eps);
#pragma unroll
    for (int j = 0; j < MAX_PER_LANE; ++j) {
      const int d = lane + 32 * j;
      if (d < head_dim) v[j] = (v[j] * inv) * to_float(norm_w[head * head_dim + d]);
    }
  } else if (norm_w != nullptr) {
    const float inv = 1.0f / sqrtf(warp_sum(sq) / norm_dim + eps);
#pragma unroll
    for (int j = 0; j < MAX_PER_LANE; ++j) {
      const int d = lane + 32 * j;
      if (d < head_dim) v[j] = (v[j] * inv) * to_float(norm_w[d]);
    }
  } else if (ex.unit_norm && kind != 2) {
    const float inv = 1.0f / sqrtf(warp_sum(sq) / norm_dim + eps);
#pragma unroll
    for (int j = 0; j < MAX_PER_LANE; ++j) v[j] *= inv;
  }
  if (kind == 2) {
    const int v_dim = ex.v_dim > 0 ? ex.v_dim : head_dim;
    if (ex.v_unit) {  // dims beyond v_dim hold zeros (zero rows of the matrix, no bias there)
      const float inv = 1.0f / sqrtf(warp_sum(sq) / (float)v_dim + eps);
#pragma unroll
      for (int j = 0; j < MAX_PER_LANE; ++j) v[j] *= inv;
    }
#pragma unroll
    for (int j = 0; j < MAX_PER_LANE; ++j) {
      const int d = lane + 32 * j;
      if (d < v_dim) {
        if (ex.v_keep != nullptr) ex.v_keep[(size_t)t * ex.v_keep_stride + head * v_dim + d] = v[j];
        if (ex.v_first != nullptr)
          v[j] = (1.0f - ex.v_blend) * v[j] + ex.v_blend * ex.v_first[(size_t)t * ex.v_first_stride + head * v_dim + d];
      }
    }
  }

  float* mine = staged + warp * head_dim;
  if (kind != 2 && rope_half > 0) {
#pragma unroll
    for (int j = 0; j < MAX_PER_LANE; ++j) {
      const int d = lane + 32 * j;
      if (d < head_dim) mine[d] = v[j];
    }
    __syncwarp();
    const float2* cs = cos_sin + (size_t)t * rope_half;
#pragma unroll
    for (int j = 0; j < MAX_PER_LANE; ++j) {
      const int d = lane + 32 * j;
      if (interleaved) {
        if (d < 2 * rope_half) {
          const float2 a = cs[d >> 1];
          v[j] = (d & 1) ? mine[d - 1] * a.y + mine[d] * a.x : mine[d] * a.x - mine[d + 1] * a.y;
        }
      } else if (d < rope_half) {
        const float2 a = cs[d];
        v[j] = mine[d] * a.x - mine[d + rope_half] * a.y;
      } else if (d < 2 * rope_half) {
        const float2 a = cs[d - rope_half];
        v[j] = mine[d - rope_half] * a.y + mine[d] * a.x;
      }
    }
  }

  if (kind == 0) {
    if (temp.every > 0) {
      const float f = temp.at(pos);
#pragma unroll
      for (int j = 0; j < MAX_PER_LANE; ++j) v[j] *= f;
    }
    TQ* dst = q_out + (size_t)t * n_heads * head_dim + head * head_dim;
#pragma unroll
    for (int j = 0; j < MAX_PER_LANE; ++j) {
      const int d = lane + 32 * j;
      if (d < head_dim) dst[d] = from_float<TQ>(v[j]);
    }
  } else {
    const int block = block_table[(size_t)slot * max_blocks + pos / XRT_BLOCK_TOKENS];
    if (block < 0) return;  // the host reserves blocks before the step; nothing to write into
    TC* pool = kind == 1 ? k_pool : v_pool;
    TC* dst = pool + (((size_t)block * n_kv_heads + head) * XRT_BLOCK_TOKENS + pos % XRT_BLOCK_TOKENS) * head_dim;
#pragma unroll
    for (int j = 0; j < MAX_PER_LANE; ++j) {
      const int d = lane + 32 * j;
      if (d < head_dim) dst[d] = from_float<TC>(v[j]);
    }
  }
}

// The same for head size 128 with the rotation over all of the head (or none): a lane holds four
// consecutive dims (one 16-byte load), the partner of dim d, d +- 64, sits sixteen lanes away (a
// shuffle instead of shared memory), and a block of eight warps walks all heads of one token, so a
// prompt launches one block a token instead of twelve.
__device__ __forceinline__ void store4_as(float* dst, const float (&v)[4]) {
  *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void store4_as(__nv_bfloat16* dst, const float (&v)[4]) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
  uint2 t;
  t.x = *reinterpret_cast<uint32_t*>(&a);
  t.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(dst) = t;
}

template <typename TN, typename TQ, typename TC>
__global__ void __launch_bounds__(256)
qk_rope_kv_write_128_kernel(
    TQ* __restrict__ q_out, TC* __restrict__ k_pool, TC* __restrict__ v_pool,
    const float* __restrict__ qkv, int row_stride, int k_offset, int v_offset,
    const TN* __restrict__ q_norm_w, const TN* __restrict__ k_norm_w, float eps,
    const float2* __restrict__ cos_sin, int rope_half,
    const int* __restrict__ tok_slot, const int* __restrict__ tok_pos,
    const int* __restrict__ block_table, int max_blocks,
    int n_heads, int n_kv_heads, int write_kv, const QueryTemp temp) {
  constexpr int HD = 128;
  pdl_trigger();
  // The step's arrays (slots, positions, block table) were written before the step began, and the norm
  // weights never change: they are read while the kernel before this one finishes.
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x;
  const int n_slots = n_heads + (write_kv ? 2 * n_kv_heads : 0);
  const int slot = tok_slot[t];
  const int pos = tok_pos[t];
  int block = -1;
  if (slot >= 0 && write_kv) block = block_table[(size_t)slot * max_blocks + pos / XRT_BLOCK_TOKENS];
  float qn[4] = {1.f, 1.f, 1.f, 1.f}, kn[4] = {1.f, 1.f, 1.f, 1.f};
  if (q_norm_w != nullptr) {
#pragma unroll
    for (int j = 0; j < 4; ++j) { qn[j] = to_float(q_norm_w[4 * lane + j]); kn[j] = to_float(k_norm_w[4 * lane + j]); }
  }
  const float q_factor = temp.at(pos);
  pdl_wait(qkv, q_norm_w, k_norm_w, cos_sin, tok_slot, tok_pos, block_table);
  // (cos, sin) of this lane's four pairs: dims 4 * (lane % 16) .. of the first half
  float c[4] = {1.f, 1.f, 1.f, 1.f}, sn[4] = {0.f, 0.f, 0.f, 0.f};
  if (rope_half > 0 && slot >= 0) {
    const float4* cs = reinterpret_cast<const float4*>(cos_sin + (size_t)t * rope_half + 4 * (lane & 15));
    const float4 a = cs[0], b = cs[1];
    c[0] = a.x; sn[0] = a.y; c[1] = a.z; sn[1] = a.w; c[2] = b.x; sn[2] = b.y; c[3] = b.z; sn[3] = b.w;
  }
  // A warp takes head slots warp, warp + 8, ...; it asks for the rows of up to four of them before it
  // works on the first (the rows come from the L2, and one load in flight a warp left the kernel waiting).
  constexpr int AHEAD = 4;
  for (int first = warp; first < n_slots; first += 8 * AHEAD) {
    float4 raw[AHEAD];
    if (slot >= 0) {
#pragma unroll
      for (int a = 0; a < AHEAD; ++a) {
        const int head_slot = first + 8 * a;
        if (head_slot < n_slots) {
          const int kind = head_slot < n_heads ? 0 : (head_slot < n_heads + n_kv_heads ? 1 : 2);
          const int head = head_slot - (kind == 0 ? 0 : (kind == 1 ? n_heads : n_heads + n_kv_heads));
          const float* src = qkv + (size_t)t * row_stride + (kind == 0 ? 0 : (kind == 1 ? k_offset : v_offset)) + head * HD;
          raw[a] = *reinterpret_cast<const float4*>(src + 4 * lane);
        }
      }
    }
#pragma unroll
    for (int a = 0; a < AHEAD; ++a) {
      const int head_slot = first + 8 * a;
      if (head_slot >= n_slots) break;
      const int kind = head_slot < n_heads ? 0 : (head_slot < n_heads + n_kv_heads ? 1 : 2);
      const int head = head_slot - (kind == 0 ? 0 : (kind == 1 ? n_heads : n_heads + n_kv_heads));
      float v[4];
      if (slot < 0) {  // a padding row: q is zeroed, the cache is not touched
        if (kind == 0) {
          v[0] = v[1] = v[2] = v[3] = 0.f;
          store4_as(q_out + (size_t)t * n_heads * HD + head * HD + 4 * lane, v);
        }
        continue;
      }
      v[0] = raw[a].x; v[1] = raw[a].y; v[2] = raw[a].z; v[3] = raw[a].w;
      const TN* norm_w = kind == 0 ? q_norm_w : (kind == 1 ? k_norm_w : nullptr);
      if (norm_w != nullptr) {
        float sq = 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) sq = fmaf(v[j], v[j], sq);
        const float inv = 1.0f / sqrtf(warp_sum(sq) / (float)HD + eps);
#pragma unroll
        for (int j = 0; j < 4; ++j) v[j] = (v[j] * inv) * (kind == 0 ? qn[j] : kn[j]);
      }
      if (kind != 2 && rope_half > 0) {
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float other = __shfl_xor_sync(0xffffffffu, v[j], 16);
          // first half: x0 cos - x1 sin; second half: x0 sin + x1 cos, with x0 the first-half element
          v[j] = lane < 16 ? v[j] * c[j] - other * sn[j] : other * sn[j] + v[j] * c[j];
        }
      }
      if (kind == 0) {
        if (temp.every > 0) {
#pragma unroll
          for (int j = 0; j < 4; ++j) v[j] *= q_factor;
        }
        store4_as(q_out + (size_t)t * n_heads * HD + head * HD + 4 * lane, v);
      } else if (block >= 0) {  // the host reserves blocks before the step; otherwise nothing to write into
        TC* pool = kind == 1 ? k_pool : v_pool;
        store4_as(pool + (((size_t)block * n_kv_heads + head) * XRT_BLOCK_TOKENS + pos % XRT_BLOCK_TOKENS) * HD + 4 * lane, v);
      }
    }
  }
}

}  // namespace xrt


XRT_EXPORT int xrt_rope_table(float* cos_sin, const int* pos, const float* freq, float scale, int n_tokens,
                              int half, cudaStream_t stream) {
  if (n_tokens < 0 || half < 0) return XRT_ERR_ARGUMENT;
  const int total = n_tokens * half;
  if (total == 0) return XRT_OK;
  xrt::launch_kernel(xrt::rope_table_kernel, dim3((total + 255) / 256), dim3(256), 0, stream, (float2*)cos_sin, pos, freq,
                     scale, n_tokens, half);
  return xrt::launch_status();
}

// freq_lo may be null (the angle is then the 32-bit product alone).
XRT_EXPORT int xrt_rotation_table(float* cos_sin, const int* pos, const float* freq, const float* freq_lo, float magnitude,
                                  int n_tokens, int half, cudaStream_t stream) {
  if (n_tokens < 0 || half < 0) return XRT_ERR_ARGUMENT;
  const int total = n_tokens * half;
  if (total == 0) return XRT_OK;
  xrt::launch_kernel(xrt::rotation_table_kernel, dim3((total + 255) / 256), dim3(256), 0, stream, (float2*)cos_sin, pos,
                     freq, freq_lo, magnitude, n_tokens, half);
  return xrt::launch_status();
}

// qkv: 32-bit rows of `row_stride` floats holding q at 0, k at k_offset, v at v_offset.
// q_out: [n_tokens, n_heads * head_dim] in q_dtype.  k_pool / v_pool: the cache blocks of this
// layer, [n_blocks, n_kv_heads, 64, head_dim] in cache_dtype.  v_offset may equal k_offset: the values are then the
// projected keys as they stand before norm and rotation.  Norm weights may be null (no head
// norm) and share norm_dtype.  write_kv = 0 leaves the cache alone (a layer reading another's).
static int qk_rope_kv_write(void* q_out, void* k_pool, void* v_pool, const float* qkv, int row_stride,
                            int k_offset, int v_offset, const void* q_norm_w, const void* k_norm_w,
                            float eps, const float* cos_sin, int rope_half, const int* tok_slot,
                            const int* tok_pos, const int* block_table, int max_blocks, int n_tokens,
                            int n_heads, int n_kv_heads, int head_dim, int write_kv, int interleaved,
                            int norm_dtype, int q_dtype, int cache_dtype, const xrt::QueryTemp& temp, const xrt::HeadExtras& ex,
                            cudaStream_t stream) {
  const bool plain = ex.bias == nullptr && !ex.unit_norm && ex.norm_dim == 0 && ex.v_keep == nullptr && ex.v_first == nullptr &&
                     ex.whole_q == 0 && ex.whole_k == 0 && !ex.v_unit;
  if (n_tokens < 0 || n_heads <= 0 || n_kv_heads <= 0 || head_dim <= 0) return XRT_ERR_ARGUMENT;
  if (head_dim > 256 || 2 * rope_half > head_dim) return XRT_ERR_UNSUPPORTED;
  if (write_kv && (q_norm_w == nullptr) != (k_norm_w == nullptr)) return XRT_ERR_ARGUMENT;  // a layer that reads another's keys norms only q
  if (n_tokens == 0) return XRT_OK;
  const bool fast = plain && head_dim == 128 && (rope_half == 0 || (rope_half == 64 && !interleaved)) && row_stride % 4 == 0 && k_offset % 4 == 0 &&
                    v_offset % 4 == 0 &&
                    (((uintptr_t)qkv | (uintptr_t)q_out | (uintptr_t)k_pool | (uintptr_t)v_pool | (uintptr_t)cos_sin) & 15) == 0;
  if (fast) {
    XRT_DISPATCH_DTYPE(norm_dtype, TN, {
      XRT_DISPATCH_DTYPE(q_dtype, TQ, {
        XRT_DISPATCH_DTYPE(cache_dtype, TC, {
          xrt::launch_kernel(xrt::qk_rope_kv_write_128_kernel<TN, TQ, TC>, dim3(n_tokens), dim3(256), 0, stream,
              (TQ*)q_out, (TC*)k_pool, (TC*)v_pool, qkv, row_stride, k_offset, v_offset, (const TN*)q_norm_w,
              (const TN*)k_norm_w, eps, (const float2*)cos_sin, rope_half, tok_slot, tok_pos, block_table,
              max_blocks, n_heads, n_kv_heads, write_kv, temp);
        });
      });
    });
    return xrt::launch_status();
  }
  const int warps = 4;
  const int n_slots = n_heads + (write_kv ? 2 * n_kv_heads : 0);
  dim3 grid(n_tokens, (n_slots + warps - 1) / warps);
  const size_t smem = (size_t)warps * head_dim * sizeof(float);
  XRT_DISPATCH_DTYPE(norm_dtype, TN, {
    XRT_DISPATCH_DTYPE(q_dtype, TQ, {
      XRT_DISPATCH_DTYPE(cache_dtype, TC, {
        xrt::launch_kernel(xrt::qk_rope_kv_write_kernel<TN, TQ, TC, 8>, grid, dim3(warps * 32), smem, stream,
            (TQ*)q_out, (TC*)k_pool, (TC*)v_pool, qkv, row_stride, k_offset, v_offset, (const TN*)q_norm_w,
            (const TN*)k_norm_w, eps, (const float2*)cos_sin, rope_half, tok_slot, tok_pos, block_table,
            max_blocks, n_heads, n_kv_heads, head_dim, write_kv, interleaved, temp, ex);
      });
    });
  });
  return xrt::launch_status();
}

XRT_EXPORT int xrt_qk_rope_kv_write(void* q_out, void* k_pool, void* v_pool, const float* qkv, int row_stride,
                                    int k_offset, int v_offset, const void* q_norm_w, const void* k_norm_w,
                                    float eps, const float* cos_sin, int rope_half, const int* tok_slot,
                                    const int* tok_pos, const int* block_table, int max_blocks, int n_tokens,
                                    int n_heads, int n_kv_heads, int head_dim, int write_kv, int interleaved,
                                    int norm_dtype, int q_dtype, int cache_dtype, float temp_coef, int temp_every,
                                    cudaStream_t stream) {
  return qk_rope_kv_write(q_out, k_pool, v_pool, qkv, row_stride, k_offset, v_offset, q_norm_w, k_norm_w, eps, cos_sin,
                          rope_half, tok_slot, tok_pos, block_table, max_blocks, n_tokens, n_heads, n_kv_heads, head_dim,
                          write_kv, interleaved, norm_dtype, q_dtype, cache_dtype, xrt::query_temp(temp_coef, temp_every),
                          xrt::HeadExtras(), stream);
}

// The same with a bias a column, weightless unit norms of q and k, norms over the whole projection, and values that
// are kept in 32-bit and / or blended with another layer's values of the same tokens before they are cached (see
// HeadExtras).
XRT_EXPORT int xrt_qkv_heads_write(void* q_out, void* k_pool, void* v_pool, const float* qkv, int row_stride,
                                   int k_offset, int v_offset, const float* bias, int unit_norm, int norm_dim, float eps,
                                   const void* q_norm_w, const void* k_norm_w, int norm_dtype, int whole_q, int whole_k,
                                   const float* cos_sin, int rope_half, int interleaved,
                                   float* v_keep, int v_keep_stride, const float* v_first, int v_first_stride,
                                   float v_blend, int v_dim, int v_unit, const int* tok_slot, const int* tok_pos,
                                   const int* block_table,
                                   int max_blocks, int n_tokens, int n_heads, int n_kv_heads, int head_dim, int write_kv,
                                   int q_dtype, int cache_dtype, float temp_coef, int temp_every, cudaStream_t stream) {
  xrt::HeadExtras ex;
  ex.v_unit = v_unit;
  ex.bias = bias;
  ex.unit_norm = unit_norm;
  ex.norm_dim = norm_dim;
  ex.v_keep = v_keep;
  ex.v_keep_stride = v_keep_stride;
  ex.v_first = v_first;
  ex.v_first_stride = v_first_stride;
  ex.v_blend = v_blend;
  ex.v_dim = v_dim;
  ex.whole_q = whole_q;
  ex.whole_k = whole_k;
  return qk_rope_kv_write(q_out, k_pool, v_pool, qkv, row_stride, k_offset, v_offset, q_norm_w, k_norm_w, eps, cos_sin,
                          rope_half, tok_slot, tok_pos, block_table, max_blocks, n_tokens, n_heads, n_kv_heads, head_dim,
                          write_kv, interleaved, norm_dtype, q_dtype, cache_dtype, xrt::query_temp(temp_coef, temp_every), ex, stream);
}
