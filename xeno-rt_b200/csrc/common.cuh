// Shared helpers of the sm_100a kernels: dtype codes, conversions, status codes, reductions.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <stdlib.h>

// dtype codes, the same integers as DType.code on the Python side
#define XRT_F32 0
#define XRT_BF16 1

// Tokens in one block of the cache; the attention kernels tile keys by it.
#define XRT_BLOCK_TOKENS 64

// Status codes returned by every launcher.  0 = launched; negative = the arguments were refused
// before any launch; positive = a cudaError_t reported by the launch.
#define XRT_OK 0
#define XRT_ERR_ARGUMENT -1
#define XRT_ERR_UNSUPPORTED -2

#define XRT_EXPORT extern "C" __attribute__((visibility("default")))

namespace xrt {

// Kernel variants a caller may force (tuning.cu holds the one instance; xrt_set_tuning sets it).
struct Tuning {
  bool pdl = true;                  // launch with programmatic dependent launch
  int decode_attention = 0;         // 0 auto, 1 heads as rows, 2 cp.async copies, 3 no clusters
  int gemm_tile_rows = 0;           // 0 auto, 128 or 256: the prefill product's tile
  bool decode_gemm_clusters = true; // the decode product's splits meet through a cluster's shared memory
  int decode_cluster_pairs = 128;    // decode attention merges its splits as clusters up to so many (token, kv head) pairs
};
const Tuning& tuning();

// A norm that is finished by the product after it.  A product that adds into the residual stream can
// prepare the RMSNorm that follows (crates/xrt-kernels/src/cpu/rmsnorm.rs:26-43), so that no norm kernel
// has to run between two products: beside the new residual it writes residual * norm weight in bfloat16
// (the next product's operand) and, for every row, partial sums of squares of the new residual (NormEmit:
// `squares` is [parts, rows]; what a part covers is the emitting kernel's business).  The next product
// multiplies row m of its result by 1 / sqrt(sum of the row's parts / width + eps) (RowScale), since
// W . ((x * inv) * w) = inv * (W . (x * w)).  The statistics are 32-bit sums over the 32-bit residual,
// added in a fixed order.
struct NormEmit {
  __nv_bfloat16* scaled = nullptr;  // [M, ld] bfloat16: new residual * weight
  const void* weight = nullptr;     // [N] norm weight, 32-bit or bfloat16
  float* squares = nullptr;         // [parts, M]
  int ld = 0;
  int weight_dtype = XRT_F32;
};
struct RowScale {
  const float* squares = nullptr;   // [parts, M], or null: the input is what it is
  int parts = 0;
  int width = 1;
  float eps = 0.f;
  // of a gated product (mode 2): 0 silu, 1 the tanh form of gelu, 2 a limited gate: with g = min(g, limit) and
  // u = clamp(u, -limit, limit) the result is g * sigmoid(alpha g) * (u + 1)
  int gate_act = 0;
  float gate_limit = 0.f, gate_alpha = 0.f;
  const float* gate_bias = nullptr; // or [gate rows | up rows]: added to both sums before the gate
  int gate_up = 0;                  // where the up rows' biases begin
};

// What a caller of a gated product may add to its mode: biases and the constants of the limited gate (null: none).
struct GateOptions {
  const float* bias;  // float32 [2 * N]: the N gate rows', then the N up rows'
  float limit, alpha;
};

// The launchers take the gate's activation in the bits of `mode` above the low four: mode 2 | (act << 4).
inline bool split_gate_act(int& mode, RowScale& scale) {
  scale.gate_act = mode >> 4;
  mode &= 15;
  return scale.gate_act == 0 || (scale.gate_act <= 2 && mode == 2);
}
inline bool take_gate_options(const GateOptions* gate, int mode, int n, RowScale& scale) {
  if (gate == nullptr) return scale.gate_act != 2;  // the limited gate has constants
  if (mode != 2) return false;
  scale.gate_bias = gate->bias;
  scale.gate_up = n;
  scale.gate_limit = gate->limit;
  scale.gate_alpha = gate->alpha;
  return true;
}

// What an attention layer may do to its scores beside the scale, the causal bound and the window (0 = off):
// keys [0, keep_first) stay visible behind a window; s <- softcap * tanh(s / softcap); then
// s <- s - slope_h * (query position - key position), slope_h = 2^(-distance_rate * (h + 1) / n_heads).
struct ScoreOptions {
  int keep_first = 0;
  float softcap = 0.f;
  float distance_rate = 0.f;
  int sink = 0;            // the softmax's denominator holds one more term exp(sink_score) that has no value
  float sink_score = 0.f;
  const float* sinks = nullptr;  // [n_heads], with sink: a head's own score instead of sink_score
};

__device__ __forceinline__ float sink_of(const ScoreOptions& opt, int head) {
  return opt.sinks != nullptr ? opt.sinks[head] : opt.sink_score;
}

// Which keys at or before its own position a query sees (0 = no such bound): the `window` most recent ones, or those
// of its own chunk of `chunk` positions, counted from position 0 of the sequence.  first(pos) never falls as pos grows,
// so the range of a tile of queries begins where its first query's does.
struct KeyRange {
  int window = 0;
  int chunk = 0;
  __host__ __device__ __forceinline__ bool bounded() const { return window > 0 || chunk > 0; }
  __device__ __forceinline__ int first(int pos) const {
    int lo = 0;
    if (window > 0) lo = max(0, pos + 1 - window);
    if (chunk > 0) lo = max(lo, pos - pos % chunk);
    return lo;
  }
};

// A temperature of the queries that grows with the logarithm of the position (every = 0: none): q at position p is
// multiplied by 1 + coef * ln(floor((p + 1) / every) + 1), 32-bit, after its norm and rotation.
struct QueryTemp {
  float coef = 0.f;
  int every = 0;
  __device__ __forceinline__ float at(int pos) const {
    return every > 0 ? fmaf(coef, logf((float)((pos + 1) / every + 1)), 1.0f) : 1.0f;
  }
};

inline QueryTemp query_temp(float coef, int every) {
  QueryTemp temp;
  temp.coef = coef;
  temp.every = every > 0 ? every : 0;
  return temp;
}

inline KeyRange key_range(int window, int chunk) {
  KeyRange range;
  range.window = window;
  range.chunk = chunk;
  return range;
}

__device__ __forceinline__ float to_float(float v) { return v; }
__device__ __forceinline__ float to_float(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T> __device__ __forceinline__ T from_float(float v);
template <> __device__ __forceinline__ float from_float<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_float<__nv_bfloat16>(float v) {
  return __float2bfloat16_rn(v);
}

// The gate of a gated feed-forward: silu, or (act 1) 0.5 g (1 + tanh(sqrt(2 / pi) (g + 0.044715 g^3))).
__device__ __forceinline__ float gelu_tanh_gate(float g) {
  return 0.5f * g * (1.0f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g)));
}

// x * sigmoid(alpha x) for a result of type TO.  A bfloat16 result keeps 8 bits: the fast exponential and
// division (2 ulp of 32-bit each) change none of them, and are a tenth of the instructions, which is
// what an epilogue that runs once a block pays for (its code comes cold from the L2).
template <typename TO> __device__ __forceinline__ float swish_for(float x, float alpha) { return x / (1.0f + expf(-alpha * x)); }
template <> __device__ __forceinline__ float swish_for<__nv_bfloat16>(float x, float alpha) {
  return __fdividef(x, 1.0f + __expf(-alpha * x));
}

// COUNT hidden units of a gated feed-forward from the two sums of their row pairs, as RowScale says, into g: units n,
// n + 1, .. with ALONG, else COUNT times unit n (of several tokens).  The kind of gate is chosen once for all of them, so
// that their exponentials and divisions run side by side.  Units at or beyond gate_up (with biases: the product's
// width) are not stored by anybody: they get some other unit's biases.
template <typename TO, int COUNT, bool ALONG>
__device__ __forceinline__ void gated_units(float (&g)[COUNT], float (&u)[COUNT], int n, const RowScale& s) {
  if (s.gate_bias != nullptr) {
    const float* up = s.gate_bias + s.gate_up;
    if (!ALONG) {
      const float bg = __ldg(s.gate_bias + n), bu = __ldg(up + n);
#pragma unroll
      for (int j = 0; j < COUNT; ++j) { g[j] += bg; u[j] += bu; }
    } else if (COUNT % 4 == 0 && ((n | s.gate_up) & 3) == 0 && ((uintptr_t)s.gate_bias & 15) == 0) {
#pragma unroll
      for (int j = 0; j + 3 < COUNT; j += 4) {
        const int at = min(n + j, s.gate_up - 4);
        const float4 bg = __ldg(reinterpret_cast<const float4*>(s.gate_bias + at));
        const float4 bu = __ldg(reinterpret_cast<const float4*>(up + at));
        g[j] += bg.x; g[j + 1] += bg.y; g[j + 2] += bg.z; g[j + 3] += bg.w;
        u[j] += bu.x; u[j + 1] += bu.y; u[j + 2] += bu.z; u[j + 3] += bu.w;
      }
    } else {
#pragma unroll
      for (int j = 0; j < COUNT; ++j) {
        const int at = min(n + j, s.gate_up - 1);
        g[j] += __ldg(s.gate_bias + at);
        u[j] += __ldg(up + at);
      }
    }
  }
  if (s.gate_act == 2) {
    const float limit = s.gate_limit, alpha = s.gate_alpha;
#pragma unroll
    for (int j = 0; j < COUNT; ++j)
      g[j] = swish_for<TO>(fminf(g[j], limit), alpha) * (fminf(fmaxf(u[j], -limit), limit) + 1.0f);
  } else if (s.gate_act == 1) {
#pragma unroll
    for (int j = 0; j < COUNT; ++j) g[j] = gelu_tanh_gate(g[j]) * u[j];
  } else {
#pragma unroll
    for (int j = 0; j < COUNT; ++j) g[j] = swish_for<TO>(g[j], 1.0f) * u[j];
  }
}

template <typename TO>
__device__ __forceinline__ float gated_unit(float g, float u, int n, const RowScale& s) {
  float gs[1] = {g}, us[1] = {u};
  gated_units<TO, 1, false>(gs, us, n, s);
  return gs[0];
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}

// Sum over a thread block with a fixed order: lanes by butterfly, then warps in index order.
// `scratch` holds at least 33 floats of shared memory.  Every thread gets the total.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int n_warps = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  if (threadIdx.x == 0) {
    float total = 0.f;
    for (int w = 0; w < n_warps; ++w) total += scratch[w];
    scratch[32] = total;
  }
  __syncthreads();
  return scratch[32];
}

// Programmatic dependent launch.  A kernel launched with `pdl` may begin while the kernel before it
// in the stream is still running: what it does before pdl_wait() (prefetching weights, set-up)
// overlaps the predecessor's tail and hides its own launch latency; pdl_wait() returns once the
// predecessor has completed and its writes are visible.  Every kernel of the decode step calls
// pdl_trigger() first (its successor may be launched) and pdl_wait() before it touches anything a
// predecessor wrote or reads anything it will overwrite.  Tuning::pdl = false turns the launch
// attribute off (the instructions are then no-ops).
__device__ __forceinline__ void pdl_trigger() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }

// The wait, for a kernel with `const T* __restrict__` parameters: such a parameter tells the compiler that what it points
// to never changes while the kernel runs, so that it may move a load through it ahead of the wait, to where the kernel
// before has not written yet.  The pointers are named here and come out of the wait as values of unknown origin: loads
// written after the wait stay after it.  (Loads written before it, of what no kernel of the step writes, stay before.)
template <typename P>
__device__ __forceinline__ void forget_origin(P& pointer) { asm volatile("" : "+l"(pointer)::"memory"); }
template <typename... P>
__device__ __forceinline__ void pdl_wait(P&... pointers) {
  asm volatile("griddepcontrol.wait;" ::: "memory");
  (forget_origin(pointers), ...);
}

inline bool pdl_enabled() { return tuning().pdl; }

template <typename... KArgs, typename... Args>
inline void launch_kernel(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                          Args... args) {
  cudaLaunchConfig_t config = {};
  config.gridDim = grid;
  config.blockDim = block;
  config.dynamicSmemBytes = smem;
  config.stream = stream;
  cudaLaunchAttribute attribute[1];
  attribute[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attribute[0].val.programmaticStreamSerializationAllowed = 1;
  const bool pdl = pdl_enabled();
  config.attrs = pdl ? attribute : nullptr;
  config.numAttrs = pdl ? 1 : 0;
  cudaLaunchKernelEx(&config, kernel, static_cast<KArgs>(args)...);
}

// A launch that waits for the kernel before it as a whole: for few blocks that run long.  Launched early, such blocks
// would be placed where the kernel before leaves room first, several on one multiprocessor while others stay empty
// (measured: twice the time for the scans of a prompt).
template <typename... KArgs, typename... Args>
inline void launch_kernel_alone(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                                Args... args) {
  cudaLaunchConfig_t config = {};
  config.gridDim = grid;
  config.blockDim = block;
  config.dynamicSmemBytes = smem;
  config.stream = stream;
  cudaLaunchKernelEx(&config, kernel, static_cast<KArgs>(args)...);
}

// The same launch with a range of global memory that the kernel reads once (a weight): its lines
// are marked as streaming in the L2 (an access-policy window of the launch), so they are the first to
// leave and what the step reads again stays.  For kernels whose copies cannot carry a cache hint
// themselves.  The window is cut to what the device allows.
template <typename... KArgs, typename... Args>
inline void launch_kernel_streaming(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                                    const void* read_once, size_t read_once_bytes, Args... args) {
  static int max_window = -1;
  if (max_window < 0) {
    int device = 0, value = 0;
    if (cudaGetDevice(&device) != cudaSuccess ||
        cudaDeviceGetAttribute(&value, cudaDevAttrMaxAccessPolicyWindowSize, device) != cudaSuccess)
      value = 0;
    cudaGetLastError();
    max_window = value;
  }
  cudaLaunchConfig_t config = {};
  config.gridDim = grid;
  config.blockDim = block;
  config.dynamicSmemBytes = smem;
  config.stream = stream;
  cudaLaunchAttribute attribute[2];
  int n = 0;
  if (pdl_enabled()) {
    attribute[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attribute[n].val.programmaticStreamSerializationAllowed = 1;
    ++n;
  }
  if (max_window > 0 && read_once != nullptr && read_once_bytes > 0) {
    attribute[n].id = cudaLaunchAttributeAccessPolicyWindow;
    attribute[n].val.accessPolicyWindow.base_ptr = const_cast<void*>(read_once);
    attribute[n].val.accessPolicyWindow.num_bytes = read_once_bytes < (size_t)max_window ? read_once_bytes : (size_t)max_window;
    attribute[n].val.accessPolicyWindow.hitRatio = 1.0f;
    attribute[n].val.accessPolicyWindow.hitProp = cudaAccessPropertyStreaming;
    attribute[n].val.accessPolicyWindow.missProp = cudaAccessPropertyStreaming;
    ++n;
  }
  config.attrs = n ? attribute : nullptr;
  config.numAttrs = n;
  cudaLaunchKernelEx(&config, kernel, static_cast<KArgs>(args)...);
}

inline int launch_status() {
  cudaError_t err = cudaPeekAtLastError();
  return err == cudaSuccess ? XRT_OK : (int)err;
}

}  // namespace xrt

// Dispatch on a dtype code: runs BODY with `T` bound to float or __nv_bfloat16.
#define XRT_DISPATCH_DTYPE(code, T, ...)            \
  do {                                              \
    if ((code) == XRT_F32) {                        \
      using T = float;                              \
      __VA_ARGS__                                   \
    } else if ((code) == XRT_BF16) {                \
      using T = __nv_bfloat16;                      \
      __VA_ARGS__                                   \
    } else {                                        \
      return XRT_ERR_UNSUPPORTED;                   \
    }                                               \
  } while (0)
