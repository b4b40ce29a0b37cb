// What a sublayer gives is added into the 32-bit residual stream, for layers that norm only what a sublayer reads:
//
//   residual[t] += factor * sum_p s_p N_p(part_p[t]),    then, if asked,   out[t] = RMSNorm(residual[t]) * w2
//
// out being the norm that the next sublayer begins with, in the compute dtype.  The parts are added in index order, so
// the sum has one order whatever else is in the step.
//   part_p[t]  row t of part p of y [parts, T, width]; or, with `rows`, row rows[t * parts + p] of y [any, width] (the
//              experts' results sorted by expert, read where they lie)
//   s_p        1, or row_scales[t * parts + p] (the experts' weights of a token), or scales[p]
//   N_p        nothing, or (part_norms, [parts, width]) RMSNorm with that part's own weight: mixers side by side whose
//              results are normed one by one before they are averaged
// Statistics, divisions and sums are 32-bit.  One block a row, V neighbouring columns a load.
#include "common.cuh"

namespace xrt {

struct StreamAdd {
  float* residual;
  const float* y;
  size_t part_stride;
  int n_parts;
  const int* rows;
  const float *row_scales, *scales;
  const float* part_norms;
  float part_eps, factor;
  const void* then_w;
  void* then_out;
  float then_eps;
  int width;
};

template <int V>
__device__ __forceinline__ void sa_load(const float* p, float (&v)[V]) {
  if constexpr (V == 4) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
  } else {
    v[0] = p[0];
  }
}

template <typename TW, typename TO, int V, int CHUNKS>
__global__ void __launch_bounds__(512) stream_add_kernel(const StreamAdd a) {
  __shared__ float scratch[33];
  pdl_trigger();
  const int width = a.width, t = blockIdx.x;
  const TW* w2 = static_cast<const TW*>(a.then_w);
  float wv[CHUNKS][V];
  if (w2 != nullptr) {  // the weight does not depend on the step: on its way while the kernel before finishes
#pragma unroll
    for (int i = 0; i < CHUNKS; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * V;
#pragma unroll
      for (int x = 0; x < V; ++x) wv[i][x] = c < width ? to_float(w2[c + x]) : 0.f;
    }
  }
  pdl_wait();
  float* r = a.residual + (size_t)t * width;
  float res[CHUNKS][V], sum[CHUNKS][V];
#pragma unroll
  for (int i = 0; i < CHUNKS; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * V;
#pragma unroll
    for (int x = 0; x < V; ++x) res[i][x] = sum[i][x] = 0.f;
    if (c < width) sa_load<V>(r + c, res[i]);
  }
  if (a.part_norms != nullptr) {
    for (int p = 0; p < a.n_parts; ++p) {
      const float* row = a.y + p * a.part_stride + (size_t)t * width;
      const float* w = a.part_norms + (size_t)p * width;
      float v[CHUNKS][V];
      float squares = 0.f;
#pragma unroll
      for (int i = 0; i < CHUNKS; ++i) {
        const int c = (threadIdx.x + i * blockDim.x) * V;
#pragma unroll
        for (int x = 0; x < V; ++x) v[i][x] = 0.f;
        if (c < width) sa_load<V>(row + c, v[i]);
      }
#pragma unroll
      for (int i = 0; i < CHUNKS; ++i)
#pragma unroll
        for (int x = 0; x < V; ++x) squares = fmaf(v[i][x], v[i][x], squares);
      const float inv = 1.0f / sqrtf(block_sum(squares, scratch) / (float)width + a.part_eps);
      const float s = a.scales != nullptr ? a.scales[p] : 1.0f;
#pragma unroll
      for (int i = 0; i < CHUNKS; ++i) {
        const int c = (threadIdx.x + i * blockDim.x) * V;
        if (c < width) {
          float wp[V];
          sa_load<V>(w + c, wp);
#pragma unroll
          for (int x = 0; x < V; ++x) sum[i][x] = fmaf((v[i][x] * inv) * wp[x], s, sum[i][x]);
        }
      }
    }
  } else {
#pragma unroll 4
    for (int p = 0; p < a.n_parts; ++p) {
      const float* row = a.rows != nullptr ? a.y + (size_t)a.rows[(size_t)t * a.n_parts + p] * width
                                           : a.y + p * a.part_stride + (size_t)t * width;
      float s = 1.0f;
      if (a.row_scales != nullptr) s = a.row_scales[(size_t)t * a.n_parts + p];
      else if (a.scales != nullptr) s = a.scales[p];
#pragma unroll
      for (int i = 0; i < CHUNKS; ++i) {
        const int c = (threadIdx.x + i * blockDim.x) * V;
        if (c < width) {
          float v[V];
          sa_load<V>(row + c, v);
#pragma unroll
          for (int x = 0; x < V; ++x) sum[i][x] = fmaf(v[x], s, sum[i][x]);
        }
      }
    }
  }
  float squares = 0.f;
#pragma unroll
  for (int i = 0; i < CHUNKS; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * V;
    if (c < width) {
#pragma unroll
      for (int x = 0; x < V; ++x) {
        res[i][x] = fmaf(a.factor, sum[i][x], res[i][x]);
        squares = fmaf(res[i][x], res[i][x], squares);
      }
      if constexpr (V == 4) *reinterpret_cast<float4*>(r + c) = make_float4(res[i][0], res[i][1], res[i][2], res[i][3]);
      else r[c] = res[i][0];
    }
  }
  if (a.then_out == nullptr) return;  // uniform over the grid
  const float inv = 1.0f / sqrtf(block_sum(squares, scratch) / (float)width + a.then_eps);
  TO* out = static_cast<TO*>(a.then_out) + (size_t)t * width;
#pragma unroll
  for (int i = 0; i < CHUNKS; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * V;
    if (c < width) {
      alignas(16) TO o[V];
#pragma unroll
      for (int x = 0; x < V; ++x) o[x] = from_float<TO>((res[i][x] * inv) * wv[i][x]);
      if (V == 4 && sizeof(TO) == 2) *reinterpret_cast<uint2*>(out + c) = *reinterpret_cast<const uint2*>(o);
      else if (V == 4) *reinterpret_cast<uint4*>(out + c) = *reinterpret_cast<const uint4*>(o);
      else out[c] = o[0];
    }
  }
}

}  // namespace xrt

// residual [T, width] float32.  See the top of the file for y, rows and the scales; then_weight [width] in weight_dtype
// and then_out [T, width] in out_dtype come together or are both null.
XRT_EXPORT int xrt_stream_add(float* residual, const float* y, long long part_stride, int n_parts, const int* rows,
                              const float* row_scales, const float* scales, const float* part_norms, float part_eps,
                              float factor, const void* then_weight, void* then_out, float then_eps, int n_tokens, int width,
                              int weight_dtype, int out_dtype, cudaStream_t stream) {
  if (n_tokens < 0 || width <= 0 || n_parts <= 0 || (then_weight == nullptr) != (then_out == nullptr)) return XRT_ERR_ARGUMENT;
  if (part_norms != nullptr && (rows != nullptr || row_scales != nullptr)) return XRT_ERR_ARGUMENT;
  if (n_tokens == 0) return XRT_OK;
  xrt::StreamAdd a = {residual, y, (size_t)part_stride, n_parts, rows, row_scales, scales, part_norms, part_eps, factor,
                      then_weight, then_out, then_eps, width};
  const bool vec = width % 4 == 0 && (((uintptr_t)residual | (uintptr_t)y | (uintptr_t)part_norms | (uintptr_t)then_out) & 15) == 0;
  const int units = vec ? width / 4 : width;
  const int threads = units > 1024 ? 512 : (units > 256 ? 256 : (units > 64 ? 128 : 64));
  const int chunks = (units + threads - 1) / threads;
  if (chunks > 32) return XRT_ERR_UNSUPPORTED;
#define XRT_STREAM_ADD(VV, CC) xrt::launch_kernel(xrt::stream_add_kernel<TW, TO, VV, CC>, dim3(n_tokens), dim3(threads), 0, stream, a)
  XRT_DISPATCH_DTYPE(weight_dtype, TW, {
    XRT_DISPATCH_DTYPE(out_dtype, TO, {
      if (vec && chunks <= 2) XRT_STREAM_ADD(4, 2);
      else if (vec && chunks <= 4) XRT_STREAM_ADD(4, 4);
      else if (vec && chunks <= 8) XRT_STREAM_ADD(4, 8);
      else if (!vec && chunks <= 4) XRT_STREAM_ADD(1, 4);
      else if (!vec) XRT_STREAM_ADD(1, 32);
      else return XRT_ERR_UNSUPPORTED;
    });
  });
#undef XRT_STREAM_ADD
  return xrt::launch_status();
}
