// The scan of a matrix state with ONE decay a head, over a step's tokens; everything 32-bit.
//
//   plain:       S_t = g_t S_(t-1) + k_t v_t^T                                          o_t = S_t^T q_t
//   delta rule:  S_t = g_t S_(t-1) + k_t u_t^T,  u_t = b_t (v_t - g_t S_(t-1)^T k_t)    o_t = S_t^T q_t
//
// with S [dim, vdim] a head.  (csrc/state_mixers.cu has the scan whose decay is a vector over the key channels.)  A
// decay that is one number lets a token read the state ONCE: with a = S_(t-1)^T k_t and c = S_(t-1)^T q_t, both taken
// in one pass over the registers that hold S,
//   u_t = b_t (v_t - g_t a)        o_t = g_t c + (q_t . k_t) u_t
// so the two sums over the rows are one chain of dependent instructions instead of two, and what the lanes fetch from
// shared memory a token is k and q, without a third vector.
//
// What else the mixers do to q, k, v and the scalars on their way in happens here, a tile of tokens at a time:
//   act        silu on q, k and v
//   unit_eps   >= 0: q and k are divided by sqrt(sum(x^2) + unit_eps) a head (as one factor a token, not a pass)
//   g          a constant a head, or exp(-exp(a_log) softplus(raw + dt_bias)) of a raw value a token and head
//   b          sigmoid of a raw value a token and head
//
// A sequence is a row of cu_seqlens / seq_slot; a row with slot -1 or no tokens is skipped.  The state is kept
// [slot][head][vdim][dim].
#include "recurrence.cuh"

namespace xrt {

struct HeadScanArgs {
  float* out;
  const float *q, *k, *v;
  const float* decay;        // raw rows [tokens, heads], or null: constant
  const float* decay_const;  // [heads]
  const float *a_log, *dt_bias;
  const float* beta;         // raw rows [tokens, heads] (delta rule)
  int q_stride, k_stride, v_stride, decay_stride, beta_stride;
  float* state;
  const int *cu_seqlens, *seq_slot;
  int n_heads, heads_per_qk, dim, vdim;
  float q_scale, unit_eps;
  int act;
  int parts, cols, tile_tokens, stage_floats;
};

constexpr int HS_NUMBERS = 5;  // a token's numbers: [TT] of (decay, write factor, q . k factor, read factor), [TT] of decay * key factor

// One block of 128 threads (whole warps at least): one sequence, one head, `cols` value columns.  PARTS neighbouring
// lanes hold C2 columns of the state between them, R rows each (every PARTS-th group of four rows, so that the lanes of
// a column read neighbouring 16 bytes); what a lane fetches of k and q serves its C2 columns.  VEC: 16-byte copies.
template <int R, int C2, bool DELTA, bool VEC>
__global__ void __launch_bounds__(128) head_scan_kernel(const HeadScanArgs a) {
  extern __shared__ float4 tile4[];
  float* tile = reinterpret_cast<float*>(tile4);
  pdl_trigger();
  const int parts = a.parts, cols = a.cols, TT = a.tile_tokens, dim = a.dim, vdim = a.vdim;
  const int padded = parts * R;
  // a stage: q | k, each [TT][padded]; v [TT][cols]; raw decays and raw betas, [TT] each (regions of whole 16 bytes); after
  // the two stages the tile's numbers
  const int vec_floats = TT * padded, v_floats = (TT * cols + 3) & ~3, tt_floats = (TT + 3) & ~3;
  float4* num = reinterpret_cast<float4*>(tile + 2 * a.stage_floats);
  float* num_seen = reinterpret_cast<float*>(num + TT);
  if (padded != dim || vdim % cols != 0)  // rows and columns beyond the head's stay zero
    for (int e = threadIdx.x; e < 2 * a.stage_floats; e += blockDim.x) tile[e] = 0.f;
  const int s = blockIdx.x, h = blockIdx.y;
  const float a_rate = a.decay != nullptr ? expf(a.a_log[h]) : 0.f;
  const float dt_bias = a.decay != nullptr ? a.dt_bias[h] : 0.f;
  const float g_const = a.decay != nullptr ? 1.f : a.decay_const[h];
  pdl_wait();
  const int slot = a.seq_slot[s];
  const int begin = a.cu_seqlens[s], end = a.cu_seqlens[s + 1];
  if (slot < 0 || end <= begin) return;
  const int part = threadIdx.x % parts, jl = (threadIdx.x / parts) * C2;  // the lane's first column in the block
  const int col0 = blockIdx.z * cols;
  const int j = col0 + jl;
  const int qh = h / a.heads_per_qk;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
  constexpr int B = VEC ? 16 : 4, E = VEC ? 4 : 1;  // bytes and floats a copy
  auto row_of = [&](int i) { return 4 * ((i / 4) * parts + part) + (i & 3); };  // the lane's i-th row

  auto issue = [&](int t0, int stage) {
    float* sq = tile + stage * a.stage_floats;
    float* sk = sq + vec_floats;
    float* sv = sk + vec_floats;
    const int nt = min(TT, end - t0), per = dim / E, vper = cols / E;
    for (int e = threadIdx.x; e < nt * per; e += blockDim.x) {
      const int tt = e / per, d = (e - tt * per) * E;
      const size_t t = (size_t)(t0 + tt);
      cp_async<B>(sq + tt * padded + d, a.q + t * a.q_stride + qh * dim + d);
      cp_async<B>(sk + tt * padded + d, a.k + t * a.k_stride + qh * dim + d);
    }
    for (int e = threadIdx.x; e < nt * vper; e += blockDim.x) {
      const int tt = e / vper, c = (e - tt * vper) * E;
      if (col0 + c < vdim) cp_async<B>(sv + tt * cols + c, a.v + (size_t)(t0 + tt) * a.v_stride + h * vdim + col0 + c);
    }
    for (int tt = threadIdx.x; tt < nt; tt += blockDim.x) {
      if (a.decay != nullptr) cp_async<4>(sv + v_floats + tt, a.decay + (size_t)(t0 + tt) * a.decay_stride + h);
      if (DELTA) cp_async<4>(sv + v_floats + tt_floats + tt, a.beta + (size_t)(t0 + tt) * a.beta_stride + h);
    }
    cp_async_commit();
  };
  // silu of what this thread's own copies brought (which only it may read before the barrier)
  auto activate_own = [&](int t0, int stage) {
    float* sq = tile + stage * a.stage_floats;
    float* sk = sq + vec_floats;
    float* sv = sk + vec_floats;
    const int nt = min(TT, end - t0), per = dim / E, vper = cols / E;
    for (int e = threadIdx.x; e < nt * per; e += blockDim.x) {
      const int tt = e / per, d = (e - tt * per) * E;
#pragma unroll
      for (int x = 0; x < E; ++x) {
        sq[tt * padded + d + x] = activate(sq[tt * padded + d + x], 1);
        sk[tt * padded + d + x] = activate(sk[tt * padded + d + x], 1);
      }
    }
    for (int e = threadIdx.x; e < nt * vper; e += blockDim.x) {
      const int tt = e / vper, c = (e - tt * vper) * E;
      if (col0 + c < vdim) {
#pragma unroll
        for (int x = 0; x < E; ++x) sv[tt * cols + c + x] = activate(sv[tt * cols + c + x], 1);
      }
    }
  };

  // the state as pairs: the multiply-adds are the packed 2 x fp32 instructions (each half a true 32-bit one)
  float2 S[C2][R / 2];
  float* sp = a.state + (((size_t)slot * a.n_heads + h) * vdim + j) * dim;  // column j + c is c * dim further
  __syncthreads();  // the zero fill is done before the first copies land
  issue(begin, 0);
#pragma unroll
  for (int c = 0; c < C2; ++c) {
    const bool live = j + c < vdim;
    if (VEC) {
#pragma unroll
      for (int i = 0; i < R; i += 4) {
        float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
        if (live && row_of(i) < dim) t = *reinterpret_cast<const float4*>(sp + (size_t)c * dim + row_of(i));
        S[c][i / 2] = make_float2(t.x, t.y);
        S[c][i / 2 + 1] = make_float2(t.z, t.w);
      }
    } else {
#pragma unroll
      for (int i = 0; i < R; i += 2)
        S[c][i / 2] = make_float2((live && row_of(i) < dim) ? sp[(size_t)c * dim + row_of(i)] : 0.f,
                                  (live && row_of(i + 1) < dim) ? sp[(size_t)c * dim + row_of(i + 1)] : 0.f);
    }
  }
  int stage = 0;
  for (int t0 = begin; t0 < end; t0 += TT, stage ^= 1) {
    const int nt = min(TT, end - t0);
    if (t0 + TT < end) {
      issue(t0 + TT, stage ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    const float* sq = tile + stage * a.stage_floats;
    const float* sk = sq + vec_floats;
    const float* sv = sk + vec_floats;
    float* sg = tile + stage * a.stage_floats + 2 * vec_floats + v_floats;
    float* sb = sg + tt_floats;
    if (a.act == 1) activate_own(t0, stage);
    for (int tt = threadIdx.x; tt < nt; tt += blockDim.x) {  // by the thread whose own copies brought the raw values
      sg[tt] = a.decay != nullptr ? expf(-a_rate * softplusf_(sg[tt] + dt_bias)) : g_const;
      sb[tt] = DELTA ? sigmoidf_(sb[tt]) : 1.0f;
    }
    __syncthreads();
    // the tokens' numbers: a warp takes four tokens at a time, whose sums run side by side
    for (int first = 4 * warp; first < nt; first += 4 * n_warps) {
      float qk[4] = {}, qq[4] = {}, kk[4] = {};
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int row = min(first + x, nt - 1) * padded;
        for (int d = lane; d < padded; d += 32) {
          const float q = sq[row + d], k = sk[row + d];
          qk[x] = fmaf(q, k, qk[x]);
          qq[x] = fmaf(q, q, qq[x]);
          kk[x] = fmaf(k, k, kk[x]);
        }
      }
#pragma unroll
      for (int x = 0; x < 4; ++x) qk[x] = warp_sum(qk[x]);
      if (a.unit_eps >= 0.f) {
#pragma unroll
        for (int x = 0; x < 4; ++x) { qq[x] = warp_sum(qq[x]); kk[x] = warp_sum(kk[x]); }
      }
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        if (lane != x || first + x >= nt) continue;
        float fq = a.q_scale, fk = 1.0f;
        if (a.unit_eps >= 0.f) {
          fq = a.q_scale / sqrtf(qq[x] + a.unit_eps);
          fk = 1.0f / sqrtf(kk[x] + a.unit_eps);
        }
        const float g = sg[first + x];
        // (g, what v or its correction is multiplied by, what the write gives back to the read-out, what S^T q counts)
        num[first + x] = make_float4(g, sb[first + x] * fk, qk[x] * fq, fq * g);
        num_seen[first + x] = g * fk;  // what S^T k (k without its factor) counts in the correction
      }
    }
    __syncthreads();
    float4 kn[R / 4], qn[R / 4];  // the next token's k and q are on their way while a token is worked on
    {
      const float4* pq = reinterpret_cast<const float4*>(sq) + part;
      const float4* pk = reinterpret_cast<const float4*>(sk) + part;
#pragma unroll
      for (int i = 0; i < R / 4; ++i) { kn[i] = pk[i * parts]; qn[i] = pq[i * parts]; }
    }
    for (int tt = 0; tt < nt; ++tt) {
      const float4 n = num[tt];
      const float g = n.x, b = n.y, qk = n.z, g_read = n.w, g_seen = DELTA ? num_seen[tt] : 0.f;
      float u[C2];
#pragma unroll
      for (int c = 0; c < C2; ++c) u[c] = sv[tt * cols + jl + c];
      float2 kr[R / 2];
      float2 seen[C2][2], read[C2][2];
#pragma unroll
      for (int c = 0; c < C2; ++c) seen[c][0] = seen[c][1] = read[c][0] = read[c][1] = make_float2(0.f, 0.f);
#pragma unroll
      for (int i = 0; i < R; i += 4) {
        kr[i / 2] = make_float2(kn[i / 4].x, kn[i / 4].y);
        kr[i / 2 + 1] = make_float2(kn[i / 4].z, kn[i / 4].w);
        const float4 qq = qn[i / 4];
#pragma unroll
        for (int c = 0; c < C2; ++c) {
          if (DELTA) {
            seen[c][0] = __ffma2_rn(S[c][i / 2], kr[i / 2], seen[c][0]);
            seen[c][1] = __ffma2_rn(S[c][i / 2 + 1], kr[i / 2 + 1], seen[c][1]);
          }
          read[c][0] = __ffma2_rn(S[c][i / 2], make_float2(qq.x, qq.y), read[c][0]);
          read[c][1] = __ffma2_rn(S[c][i / 2 + 1], make_float2(qq.z, qq.w), read[c][1]);
        }
      }
      {
        // the lane's i-th group of four rows is 16-byte element i * parts of these
        const int next = min(tt + 1, nt - 1) * padded;
        const float4* pq = reinterpret_cast<const float4*>(sq + next) + part;
        const float4* pk = reinterpret_cast<const float4*>(sk + next) + part;
#pragma unroll
        for (int i = 0; i < R / 4; ++i) { kn[i] = pk[i * parts]; qn[i] = pq[i * parts]; }
      }
      float along[C2], out[C2];
#pragma unroll
      for (int c = 0; c < C2; ++c) {
        along[c] = (seen[c][0].x + seen[c][0].y) + (seen[c][1].x + seen[c][1].y);
        out[c] = (read[c][0].x + read[c][0].y) + (read[c][1].x + read[c][1].y);
      }
      for (int o = 1; o < parts; o <<= 1) {
#pragma unroll
        for (int c = 0; c < C2; ++c) {
          if (DELTA) along[c] += __shfl_xor_sync(0xffffffffu, along[c], o);
          out[c] += __shfl_xor_sync(0xffffffffu, out[c], o);
        }
      }
#pragma unroll
      for (int c = 0; c < C2; ++c) {
        u[c] = DELTA ? b * (u[c] - g_seen * along[c]) : b * u[c];
        out[c] = fmaf(g_read, out[c], qk * u[c]);
        const float2 uu = make_float2(u[c], u[c]), gg = make_float2(g, g);
#pragma unroll
        for (int i = 0; i < R / 2; ++i) S[c][i] = __ffma2_rn(S[c][i], gg, __fmul2_rn(kr[i], uu));
      }
      if (part == 0) {
        float* dst = a.out + (size_t)(t0 + tt) * a.n_heads * vdim + h * vdim + j;
#pragma unroll
        for (int c = 0; c < C2; ++c)
          if (j + c < vdim) dst[c] = out[c];
      }
    }
    __syncthreads();  // the stage and the numbers are read out before the next tile overwrites them
  }
#pragma unroll
  for (int c = 0; c < C2; ++c) {
    if (j + c >= vdim) continue;
    if (VEC) {
#pragma unroll
      for (int i = 0; i < R; i += 4)
        if (row_of(i) < dim)
          *reinterpret_cast<float4*>(sp + (size_t)c * dim + row_of(i)) =
              make_float4(S[c][i / 2].x, S[c][i / 2].y, S[c][i / 2 + 1].x, S[c][i / 2 + 1].y);
    } else {
#pragma unroll
      for (int i = 0; i < R; i += 2) {
        if (row_of(i) < dim) sp[(size_t)c * dim + row_of(i)] = S[c][i / 2].x;
        if (row_of(i + 1) < dim) sp[(size_t)c * dim + row_of(i + 1)] = S[c][i / 2].y;
      }
    }
  }
}

}  // namespace xrt

// decay: raw rows (with a_log, dt_bias), or null with decay_const [heads].  beta: raw rows, or null (no delta rule).
// unit_eps < 0: q and k as they come.  act: 0, or 1 (silu on q, k, v).  max_new (0: not known): the most tokens a
// sequence of the step brings.
XRT_EXPORT int xrt_head_scan(float* out, const float* q, int q_stride, const float* k, int k_stride, const float* v,
                             int v_stride, const float* decay, int decay_stride, const float* decay_const,
                             const float* a_log, const float* dt_bias, const float* beta, int beta_stride, float* state,
                             const int* cu_seqlens, const int* seq_slot, int n_seqs, int n_heads, int n_qk_heads, int dim,
                             int vdim, float q_scale, float unit_eps, int act, int max_new, cudaStream_t stream) {
  if (n_seqs < 0 || n_heads <= 0 || n_qk_heads <= 0 || n_heads % n_qk_heads || dim <= 0 || vdim <= 0 || (act != 0 && act != 1))
    return XRT_ERR_ARGUMENT;
  if (decay != nullptr ? (a_log == nullptr || dt_bias == nullptr) : decay_const == nullptr) return XRT_ERR_ARGUMENT;
  if (dim > 1024 || n_heads > 65535) return XRT_ERR_UNSUPPORTED;
  if (n_seqs == 0) return XRT_OK;
  if (max_new < 1) max_new = 1 << 30;
  const bool delta = beta != nullptr;
  const int R = dim <= 512 ? 16 : 32;
  int parts = 1;
  while (parts * R < dim) parts <<= 1;
  // columns a lane holds: as many as leave every multiprocessor a block (what a lane fetches of k and q then serves
  // more columns: the kernel is bound by what its warps ask of shared memory)
  int per_lane = R == 16 ? 4 : 1;
  int groups = 128 / parts;
  while (per_lane > 1 && (groups * per_lane / 2 >= vdim ||
                          (long long)n_seqs * n_heads * ((vdim + groups * per_lane - 1) / (groups * per_lane)) < 148))
    per_lane >>= 1;
  while (groups > 1 && (groups / 2) * per_lane >= vdim && (groups / 2) * parts >= 32) groups >>= 1;
  const int cols = groups * per_lane, padded = parts * R;
  auto stage_floats = [&](int tt) { return 2 * tt * padded + ((tt * cols + 3) & ~3) + 2 * ((tt + 3) & ~3); };
  auto bytes = [&](int tt) { return (2 * (size_t)stage_floats(tt) + xrt::HS_NUMBERS * tt) * sizeof(float); };
  int tile_tokens = 16;
  while (tile_tokens > 1 && bytes(tile_tokens) > 46 * 1024) tile_tokens >>= 1;
  while (tile_tokens > 1 && tile_tokens / 2 >= max_new) tile_tokens >>= 1;
  if (bytes(tile_tokens) > 48 * 1024) return XRT_ERR_UNSUPPORTED;
  const bool vec = dim % 4 == 0 && vdim % 4 == 0 && cols % 4 == 0 && q_stride % 4 == 0 && k_stride % 4 == 0 &&
                   v_stride % 4 == 0 && (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)state) & 15) == 0;
  xrt::HeadScanArgs a = {out, q, k, v, decay, decay_const, a_log, dt_bias, beta, q_stride, k_stride, v_stride, decay_stride,
                         beta_stride, state, cu_seqlens, seq_slot, n_heads, n_heads / n_qk_heads, dim, vdim, q_scale,
                         unit_eps, act, parts, cols, tile_tokens, stage_floats(tile_tokens)};
  const dim3 grid(n_seqs, n_heads, (vdim + cols - 1) / cols), block(parts * groups);
#define XRT_HEAD_SCAN(RR, CC)                                                                                           \
  do {                                                                                                                  \
    if (delta && vec) xrt::launch_kernel(xrt::head_scan_kernel<RR, CC, true, true>, grid, block, bytes(tile_tokens), stream, a);        \
    else if (delta) xrt::launch_kernel(xrt::head_scan_kernel<RR, CC, true, false>, grid, block, bytes(tile_tokens), stream, a);         \
    else if (vec) xrt::launch_kernel(xrt::head_scan_kernel<RR, CC, false, true>, grid, block, bytes(tile_tokens), stream, a);           \
    else xrt::launch_kernel(xrt::head_scan_kernel<RR, CC, false, false>, grid, block, bytes(tile_tokens), stream, a);                   \
  } while (0)
  if (R == 32) XRT_HEAD_SCAN(32, 1);
  else if (per_lane == 4) XRT_HEAD_SCAN(16, 4);
  else if (per_lane == 2) XRT_HEAD_SCAN(16, 2);
  else XRT_HEAD_SCAN(16, 1);
#undef XRT_HEAD_SCAN
  return xrt::launch_status();
}
