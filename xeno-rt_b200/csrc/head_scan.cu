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

// A lane's part of the state: C2 columns (of which `live` lie inside the head), R rows each at row_of(i), as pairs (the
// multiply-adds are the packed 2 x fp32 instructions, each half a true 32-bit one).  Column c is at sp + c * dim.
template <int R, int C2, bool VEC, typename RowOf>
__device__ __forceinline__ void load_state(float2 (&S)[C2][R / 2], const float* sp, int dim, int live, RowOf row_of) {
#pragma unroll
  for (int c = 0; c < C2; ++c) {
    if (VEC) {
#pragma unroll
      for (int i = 0; i < R; i += 4) {
        float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < live && row_of(i) < dim) t = *reinterpret_cast<const float4*>(sp + (size_t)c * dim + row_of(i));
        S[c][i / 2] = make_float2(t.x, t.y);
        S[c][i / 2 + 1] = make_float2(t.z, t.w);
      }
    } else {
#pragma unroll
      for (int i = 0; i < R; i += 2)
        S[c][i / 2] = make_float2((c < live && row_of(i) < dim) ? sp[(size_t)c * dim + row_of(i)] : 0.f,
                                  (c < live && row_of(i + 1) < dim) ? sp[(size_t)c * dim + row_of(i + 1)] : 0.f);
    }
  }
}

template <int R, int C2, bool VEC, typename RowOf>
__device__ __forceinline__ void store_state(const float2 (&S)[C2][R / 2], float* sp, int dim, int live, RowOf row_of) {
#pragma unroll
  for (int c = 0; c < C2; ++c) {
    if (c >= live) continue;
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

  float2 S[C2][R / 2];
  float* sp = a.state + (((size_t)slot * a.n_heads + h) * vdim + j) * dim;  // column j + c is c * dim further
  __syncthreads();  // the zero fill is done before the first copies land
  issue(begin, 0);
  load_state<R, C2, VEC>(S, sp, dim, vdim - j, row_of);
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
  store_state<R, C2, VEC>(S, sp, dim, vdim - j, row_of);
}

// ------------------------------------------------------------------------------------------ portions of several tokens
// Four tokens at a time.  With S the state before a group and, for its tokens i = 0 .. 3, s_i = S^T k_i and r_i = S^T q_i
// (k_i, q_i as they lie in memory, without the factors f_i, h_i of their unit norms and the read-out's scale),
//   w_i = A_i v_i - C_i s_i - sum_(j < i) M_ij w_j                 what token i writes along k_i
//   o_i = D_i r_i + sum_(j <= i) N_ij w_j                          what it reads, its own write included
//   S  <- G S + sum_j k_j (E_j w_j)
// and with g the decays, b the write factors, P(j, i) = g_(j+1) .. g_i:
//   A_i = b_i f_i   C_i = b_i f_i^2 P(-1, i)   M_ij = b_i f_i^2 P(j, i) (k_j . k_i)   (plain: A = 1, C = M = 0)
//   D_i = h_i P(-1, i)   N_ij = h_i P(j, i) (k_j . q_i)   E_j = P(j, 3)   G = P(-1, 3)
// The terms do not depend on the state: a kernel of its own makes them for all groups at once.  The scan then has eight
// independent sums over a lane's rows a group, and a chain of a dozen scalar steps, where token by token it would have
// four times the chain.  A group that the sequence ends inside is filled up with tokens that write nothing (g = 1, b = 0).
// Groups are counted from the step's first token of each sequence; group c of sequence s is row begin / 4 + s + c of the
// terms, which no other sequence's groups reach.
constexpr int HS_TERMS = 32;  // A[4] C[4] D[4] E[3] G M10 M20 M21 M30 M31 M32 N00 N10 N11 N20 N21 N22 N30 N31 N32 N33

__device__ __forceinline__ size_t group_row(int begin, int s, int c, int n_heads, int h) {
  return ((size_t)(begin / 4 + s + c) * n_heads + h) * HS_TERMS;
}

// One warp a (group, head); grid (groups of the longest sequence, heads / warps, sequences).
__global__ void __launch_bounds__(128) head_scan_terms_kernel(float* __restrict__ terms, const HeadScanArgs a) {
  pdl_trigger();
  pdl_wait();
  const int s = blockIdx.z, h = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int slot = a.seq_slot[s], begin = a.cu_seqlens[s], end = a.cu_seqlens[s + 1];
  const int t0 = begin + 4 * blockIdx.x, nt = min(4, end - t0);
  if (slot < 0 || nt <= 0 || h >= a.n_heads) return;
  const int qh = h / a.heads_per_qk;
  float kk[4][4] = {}, kq[4][4] = {}, qq[4] = {};  // kk[i][j] = k_j . k_i, kq[i][j] = k_j . q_i for j <= i
  for (int d = lane; d < a.dim; d += 32) {
    float q[4], k[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const size_t t = (size_t)(t0 + min(i, nt - 1));
      q[i] = a.q[t * a.q_stride + qh * a.dim + d];
      k[i] = a.k[t * a.k_stride + qh * a.dim + d];
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      qq[i] = fmaf(q[i], q[i], qq[i]);
#pragma unroll
      for (int j = 0; j <= i; ++j) {
        kk[i][j] = fmaf(k[i], k[j], kk[i][j]);
        kq[i][j] = fmaf(q[i], k[j], kq[i][j]);
      }
    }
  }
  float g[4], b[4], f[4], hq[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const size_t t = (size_t)(t0 + min(i, nt - 1));
    g[i] = a.decay == nullptr ? a.decay_const[h] : expf(-expf(a.a_log[h]) * softplusf_(a.decay[t * a.decay_stride + h] + a.dt_bias[h]));
    b[i] = a.beta == nullptr ? 1.0f : sigmoidf_(a.beta[t * a.beta_stride + h]);
    if (i >= nt) { g[i] = 1.0f; b[i] = 0.0f; }
#pragma unroll
    for (int j = 0; j <= i; ++j) { kk[i][j] = warp_sum(kk[i][j]); kq[i][j] = warp_sum(kq[i][j]); }
    f[i] = a.unit_eps >= 0.f ? 1.0f / sqrtf(kk[i][i] + a.unit_eps) : 1.0f;
    hq[i] = a.unit_eps >= 0.f ? a.q_scale / sqrtf(warp_sum(qq[i]) + a.unit_eps) : a.q_scale;
  }
  if (lane != 0) return;
  float out[HS_TERMS];
  float from_start = 1.0f;
  int m = 16, n = 22;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    from_start *= g[i];
    const float bff = a.beta != nullptr ? b[i] * f[i] * f[i] : 0.0f;
    out[i] = b[i] * f[i];
    out[4 + i] = bff * from_start;
    out[8 + i] = hq[i] * from_start;
#pragma unroll
    for (int j = 0; j <= i; ++j) {
      float between = 1.0f;  // P(j, i)
#pragma unroll
      for (int l = j + 1; l <= i; ++l) between *= g[l];
      if (j < i) out[m++] = bff * between * kk[i][j];
      out[n++] = hq[i] * between * kq[i][j];
    }
  }
#pragma unroll
  for (int j = 0; j < 3; ++j) {
    float after = 1.0f;
#pragma unroll
    for (int l = j + 1; l < 4; ++l) after *= g[l];
    out[12 + j] = after;
  }
  out[15] = from_start;
  float4* dst = reinterpret_cast<float4*>(terms + group_row(begin, s, blockIdx.x, a.n_heads, h));
#pragma unroll
  for (int i = 0; i < HS_TERMS / 4; ++i) dst[i] = make_float4(out[4 * i], out[4 * i + 1], out[4 * i + 2], out[4 * i + 3]);
}

// One block: one sequence, one head, `cols` value columns; PARTS neighbouring lanes hold C2 columns of the state between
// them, R rows each (as in head_scan_kernel).  A stage: q | k, each [TT][padded]; v [TT][cols]; terms [TT / 4][HS_TERMS].
template <int R, int C2, bool DELTA, bool VEC>
__global__ void __launch_bounds__(128) head_scan_groups_kernel(const float* __restrict__ terms, const HeadScanArgs a) {
  extern __shared__ float4 tile4[];
  float* tile = reinterpret_cast<float*>(tile4);
  pdl_trigger();
  const int parts = a.parts, cols = a.cols, TT = a.tile_tokens, dim = a.dim, vdim = a.vdim;
  const int padded = parts * R;
  const int vec_floats = TT * padded, v_floats = (TT * cols + 3) & ~3;
  if (padded != dim || vdim % cols != 0)  // rows and columns beyond the head's stay zero
    for (int e = threadIdx.x; e < 2 * a.stage_floats; e += blockDim.x) tile[e] = 0.f;
  pdl_wait(terms);
  const int s = blockIdx.x, h = blockIdx.y;
  const int slot = a.seq_slot[s];
  const int begin = a.cu_seqlens[s], end = a.cu_seqlens[s + 1];
  if (slot < 0 || end <= begin) return;
  const int part = threadIdx.x % parts, jl = (threadIdx.x / parts) * C2;  // the lane's first column in the block
  const int col0 = blockIdx.z * cols;
  const int j = col0 + jl;
  const int qh = h / a.heads_per_qk;
  constexpr int B = VEC ? 16 : 4, E = VEC ? 4 : 1;  // bytes and floats a copy
  auto row_of = [&](int i) { return 4 * ((i / 4) * parts + part) + (i & 3); };  // the lane's i-th row

  // a thread copies the same column(s) of every token: no division a copy
  const int per = dim / E, vper = cols / E;
  auto issue = [&](int t0, int stage) {
    float* sq = tile + stage * a.stage_floats;
    float* sk = sq + vec_floats;
    float* sv = sk + vec_floats;
    float* st = sv + v_floats;
    const int nt = min(TT, end - t0);
    const int lanes = min(per, (int)blockDim.x), rows = blockDim.x / lanes;  // threads a row, rows at a time
    const int first = threadIdx.x / lanes, at = threadIdx.x - first * lanes;
    if (first < rows)
      for (int tt = first; tt < nt; tt += rows)
        for (int e = at; e < per; e += lanes) {
          const size_t t = (size_t)(t0 + tt);
          cp_async<B>(sq + tt * padded + e * E, a.q + t * a.q_stride + qh * dim + e * E);
          cp_async<B>(sk + tt * padded + e * E, a.k + t * a.k_stride + qh * dim + e * E);
        }
    for (int e = threadIdx.x; e < nt * vper; e += blockDim.x) {
      const int tt = e / vper, c = (e - tt * vper) * E;
      if (col0 + c < vdim) cp_async<B>(sv + tt * cols + c, a.v + (size_t)(t0 + tt) * a.v_stride + h * vdim + col0 + c);
    }
    for (int e = threadIdx.x; e < ((nt + 3) / 4) * (HS_TERMS / 4); e += blockDim.x) {
      const int c = e / (HS_TERMS / 4), x = e - c * (HS_TERMS / 4);
      cp_async<16>(st + c * HS_TERMS + 4 * x, terms + group_row(begin, s, (t0 - begin) / 4 + c, a.n_heads, h) + 4 * x);
    }
    cp_async_commit();
  };

  float2 S[C2][R / 2];
  float* sp = a.state + (((size_t)slot * a.n_heads + h) * vdim + j) * dim;  // column j + c is c * dim further
  __syncthreads();  // the zero fill is done before the first copies land
  issue(begin, 0);
  load_state<R, C2, VEC>(S, sp, dim, vdim - j, row_of);
  int stage = 0;
  for (int t0 = begin; t0 < end; t0 += TT, stage ^= 1) {
    const int nt = min(TT, end - t0);
    if (t0 + TT < end) {
      issue(t0 + TT, stage ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const float* sq = tile + stage * a.stage_floats;
    const float* sk = sq + vec_floats;
    const float* sv = sk + vec_floats;
    const float* st = sv + v_floats;
    for (int tt = 0; tt < nt; tt += 4) {
      // the lane's i-th group of four rows is 16-byte element i * parts of these
      const float4 *pq[4], *pk[4];
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int row = min(tt + x, nt - 1) * padded;
        pq[x] = reinterpret_cast<const float4*>(sq + row) + part;
        pk[x] = reinterpret_cast<const float4*>(sk + row) + part;
      }
      float2 kr[4][R / 2];
      float2 seen[C2][4], read[C2][4];
#pragma unroll
      for (int c = 0; c < C2; ++c)
#pragma unroll
        for (int x = 0; x < 4; ++x) seen[c][x] = read[c][x] = make_float2(0.f, 0.f);
#pragma unroll
      for (int i = 0; i < R; i += 4) {
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const float4 kq = pk[x][(i / 4) * parts], qq = pq[x][(i / 4) * parts];
          kr[x][i / 2] = make_float2(kq.x, kq.y);
          kr[x][i / 2 + 1] = make_float2(kq.z, kq.w);
#pragma unroll
          for (int c = 0; c < C2; ++c) {
            if (DELTA) {
              seen[c][x] = __ffma2_rn(S[c][i / 2], kr[x][i / 2], seen[c][x]);
              seen[c][x] = __ffma2_rn(S[c][i / 2 + 1], kr[x][i / 2 + 1], seen[c][x]);
            }
            read[c][x] = __ffma2_rn(S[c][i / 2], make_float2(qq.x, qq.y), read[c][x]);
            read[c][x] = __ffma2_rn(S[c][i / 2 + 1], make_float2(qq.z, qq.w), read[c][x]);
          }
        }
      }
      float along[C2][4], out[C2][4];
#pragma unroll
      for (int c = 0; c < C2; ++c)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          along[c][x] = seen[c][x].x + seen[c][x].y;
          out[c][x] = read[c][x].x + read[c][x].y;
        }
      for (int o = 1; o < parts; o <<= 1) {
#pragma unroll
        for (int c = 0; c < C2; ++c)
#pragma unroll
          for (int x = 0; x < 4; ++x) {
            if (DELTA) along[c][x] += __shfl_xor_sync(0xffffffffu, along[c][x], o);
            out[c][x] += __shfl_xor_sync(0xffffffffu, out[c][x], o);
          }
      }
      const float4* ct = reinterpret_cast<const float4*>(st + (tt / 4) * HS_TERMS);
      const float4 A = ct[0], D = ct[2], E3 = ct[3];
      const float4 n0 = ct[5], n1 = ct[6], n2 = ct[7];   // (M31 M32 N00 N10) (N11 N20 N21 N22) (N30 N31 N32 N33)
      float4 C = make_float4(0.f, 0.f, 0.f, 0.f), m0 = C;  // m0 = (M10 M20 M21 M30)
      if (DELTA) { C = ct[1]; m0 = ct[4]; }
#pragma unroll
      for (int c = 0; c < C2; ++c) {
        const float* v = sv + tt * cols + jl + c;
        float w[4];
        w[0] = A.x * v[0];
        w[1] = A.y * v[min(tt + 1, nt - 1) * cols - tt * cols];
        w[2] = A.z * v[min(tt + 2, nt - 1) * cols - tt * cols];
        w[3] = A.w * v[min(tt + 3, nt - 1) * cols - tt * cols];
        if (DELTA) {
          w[0] = fmaf(-C.x, along[c][0], w[0]);
          w[1] = fmaf(-C.y, along[c][1], w[1]);
          w[2] = fmaf(-C.z, along[c][2], w[2]);
          w[3] = fmaf(-C.w, along[c][3], w[3]);
          w[1] = fmaf(-m0.x, w[0], w[1]);
          w[2] = fmaf(-m0.y, w[0], w[2]);
          w[3] = fmaf(-m0.w, w[0], w[3]);
          w[2] = fmaf(-m0.z, w[1], w[2]);
          w[3] = fmaf(-n0.x, w[1], w[3]);
          w[3] = fmaf(-n0.y, w[2], w[3]);
        }
        const float e0 = E3.x * w[0], e1 = E3.y * w[1], e2 = E3.z * w[2];
        const float2 g = make_float2(E3.w, E3.w);
#pragma unroll
        for (int i = 0; i < R / 2; ++i) {
          S[c][i] = __ffma2_rn(S[c][i], g, __fmul2_rn(kr[0][i], make_float2(e0, e0)));
          S[c][i] = __ffma2_rn(kr[1][i], make_float2(e1, e1), S[c][i]);
          S[c][i] = __ffma2_rn(kr[2][i], make_float2(e2, e2), S[c][i]);
          S[c][i] = __ffma2_rn(kr[3][i], make_float2(w[3], w[3]), S[c][i]);
        }
        out[c][0] = fmaf(D.x, out[c][0], n0.z * w[0]);
        out[c][1] = fmaf(D.y, out[c][1], fmaf(n0.w, w[0], n1.x * w[1]));
        out[c][2] = fmaf(D.z, out[c][2], fmaf(n1.y, w[0], fmaf(n1.z, w[1], n1.w * w[2])));
        out[c][3] = fmaf(D.w, out[c][3], fmaf(n2.x, w[0], fmaf(n2.y, w[1], fmaf(n2.z, w[2], n2.w * w[3]))));
      }
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        if (part != (x & (parts - 1)) || tt + x >= nt) continue;  // the lanes of a column share the tokens' stores
        float* dst = a.out + (size_t)(t0 + tt + x) * a.n_heads * vdim + h * vdim + j;
#pragma unroll
        for (int c = 0; c < C2; ++c)
          if (j + c < vdim) dst[c] = out[c][x];
      }
    }
    __syncthreads();  // the stage is read out before the copies of the tile after next overwrite it
  }
  store_state<R, C2, VEC>(S, sp, dim, vdim - j, row_of);
}

}  // namespace xrt

// decay: raw rows (with a_log, dt_bias), or null with decay_const [heads].  beta: raw rows, or null (no delta rule).
// unit_eps < 0: q and k as they come.  act: 0, or 1 (silu on q, k, v).  max_new (0: not known): the most tokens a
// sequence of the step brings.  terms (null: not given): scratch of (tokens / 4 + n_seqs + 1) * n_heads * 32 floats, 16-byte
// aligned; with it, and act 0, portions of several tokens run four tokens at a time.
XRT_EXPORT int xrt_head_scan(float* out, const float* q, int q_stride, const float* k, int k_stride, const float* v,
                             int v_stride, const float* decay, int decay_stride, const float* decay_const,
                             const float* a_log, const float* dt_bias, const float* beta, int beta_stride, float* state,
                             const int* cu_seqlens, const int* seq_slot, int n_seqs, int n_heads, int n_qk_heads, int dim,
                             int vdim, float q_scale, float unit_eps, int act, int max_new, float* terms,
                             cudaStream_t stream) {
  if (n_seqs < 0 || n_heads <= 0 || n_qk_heads <= 0 || n_heads % n_qk_heads || dim <= 0 || vdim <= 0 || (act != 0 && act != 1))
    return XRT_ERR_ARGUMENT;
  if (decay != nullptr ? (a_log == nullptr || dt_bias == nullptr) : decay_const == nullptr) return XRT_ERR_ARGUMENT;
  if (dim > 1024 || n_heads > 65535) return XRT_ERR_UNSUPPORTED;
  if (n_seqs == 0) return XRT_OK;
  const bool delta = beta != nullptr;
  if (terms != nullptr && max_new > 1 && act == 0 && dim <= 512 && n_seqs <= 65535) {  // portions: four tokens at a time
    // columns a lane: as many as leave the device full (what a lane fetches of k and q serves them all)
    const long long columns = (long long)n_seqs * n_heads * vdim;
    constexpr int R = 16;
    int per_lane = 1;
    if (columns >= 4096) per_lane = 2;
    if (columns >= 16384) per_lane = 4;
    while (per_lane > 1 && 128 / ((dim + R - 1) / R) * per_lane / 2 >= vdim) per_lane >>= 1;
    int parts = 1;
    while (parts * R < dim) parts <<= 1;
    int groups = 128 / parts;
    while (groups > 1 && (groups / 2) * per_lane >= vdim && (groups / 2) * parts >= 32) groups >>= 1;
    const int cols = groups * per_lane, padded = parts * R;
    auto stage_floats = [&](int tt) { return 2 * tt * padded + ((tt * cols + 3) & ~3) + tt / 4 * xrt::HS_TERMS; };
    int tile_tokens = 16;
    while (tile_tokens > 4 && 2 * stage_floats(tile_tokens) * sizeof(float) > 48 * 1024) tile_tokens >>= 1;
    const size_t smem = 2 * (size_t)stage_floats(tile_tokens) * sizeof(float);
    if (smem <= 48 * 1024) {
      const bool vec = dim % 4 == 0 && vdim % 4 == 0 && cols % 4 == 0 && q_stride % 4 == 0 && k_stride % 4 == 0 &&
                       v_stride % 4 == 0 && (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)state) & 15) == 0;
      xrt::HeadScanArgs a = {out, q, k, v, decay, decay_const, a_log, dt_bias, beta, q_stride, k_stride, v_stride, decay_stride,
                             beta_stride, state, cu_seqlens, seq_slot, n_heads, n_heads / n_qk_heads, dim, vdim, q_scale,
                             unit_eps, act, parts, cols, tile_tokens, stage_floats(tile_tokens)};
      xrt::launch_kernel(xrt::head_scan_terms_kernel, dim3((max_new + 3) / 4, (n_heads + 3) / 4, n_seqs), dim3(128), 0, stream,
                         terms, a);
      const dim3 grid(n_seqs, n_heads, (vdim + cols - 1) / cols), block(parts * groups);
#define XRT_GROUPS(RR, CC, DD, VV) xrt::launch_kernel_alone(xrt::head_scan_groups_kernel<RR, CC, DD, VV>, grid, block, smem, stream, terms, a)
#define XRT_GROUPS_R(RR, CC)                          \
  do {                                                \
    if (delta && vec) XRT_GROUPS(RR, CC, true, true);  \
    else if (delta) XRT_GROUPS(RR, CC, true, false);   \
    else if (vec) XRT_GROUPS(RR, CC, false, true);     \
    else XRT_GROUPS(RR, CC, false, false);             \
  } while (0)
      if (per_lane == 4) XRT_GROUPS_R(16, 4);
      else if (per_lane == 2) XRT_GROUPS_R(16, 2);
      else XRT_GROUPS_R(16, 1);
#undef XRT_GROUPS_R
#undef XRT_GROUPS
      return xrt::launch_status();
    }
  }
  if (max_new < 1) max_new = 1 << 30;
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
