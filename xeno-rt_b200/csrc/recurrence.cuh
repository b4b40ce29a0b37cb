// What the kernels of the recurrent mixers share: 32-bit activations and asynchronous copies to shared memory.
#pragma once

#include "common.cuh"

namespace xrt {

__device__ __forceinline__ float sigmoidf_(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplusf_(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float activate(float z, int act) {  // 0 none, 1 silu, 2 sigmoid, 3 tanh
  return act == 1 ? z * sigmoidf_(z) : (act == 2 ? sigmoidf_(z) : (act == 3 ? tanhf(z) : z));
}

template <int BYTES>
__device__ __forceinline__ void cp_async(float* smem, const float* global) {
  const unsigned dst = (unsigned)__cvta_generic_to_shared(smem);
  if (BYTES == 16) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(global) : "memory");
  else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(dst), "l"(global) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

}  // namespace xrt
