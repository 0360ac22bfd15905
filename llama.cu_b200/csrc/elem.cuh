// Element conversions, the gate function and the clustered launch shared by the block-model kernels.
#pragma once
#include <cuda_bf16.h>
#include <math_constants.h>

#include "common.cuh"

namespace lcu {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

__host__ __device__ __forceinline__ int round_up_dev(int a, int b) { return (a + b - 1) / b * b; }

// asks for the line of an address in L2 (no register, nothing to wait for); may run ahead of the kernel before this one,
// whatever that kernel still writes: only the line is fetched, the value is read later
__device__ __forceinline__ void l2_line(const void* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }

// the `top` largest of z[0 .. n-1] (ties: the lower index) by one warp, in descending order: emit(k, index, value); z is used up
template <typename F>
__device__ __forceinline__ void pick_largest(float* z, int n, int top, F emit) {
  const int lane = threadIdx.x & 31;
  for (int k = 0; k < top; ++k) {
    float best = -CUDART_INF_F;
    int at = n;
    for (int e = lane; e < n; e += 32)
      if (z[e] > best) {
        best = z[e];
        at = e;
      }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float b = __shfl_xor_sync(0xffffffffu, best, o);
      const int a = __shfl_xor_sync(0xffffffffu, at, o);
      if (a < n && (at >= n || b > best || (b == best && a < at))) {
        best = b;
        at = a;
      }
    }
    if (at >= n) at = 0;  // (no value compares: not a number everywhere)
    if (lane == 0) {
      emit(k, at, best);
      z[at] = -CUDART_INF_F;
    }
    __syncwarp();
  }
}
__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }

// launch of a kernel whose CTAs work in clusters of `cluster` (1: plain), as a programmatic dependent of the kernel before it
template <typename... KP, typename... Args>
int launch_clustered(void (*kernel)(KP...), int grid, int cluster, int threads, size_t smem, cudaStream_t stream, Args&&... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(grid);
  cfg.blockDim = dim3(threads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  int n = 0;
  if (cluster > 1) {
    attr[n].id = cudaLaunchAttributeClusterDimension;
    attr[n].val.clusterDim.x = cluster;
    attr[n].val.clusterDim.y = 1;
    attr[n].val.clusterDim.z = 1;
    ++n;
  }
  if (prompt_pdl()) {
    attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[n].val.programmaticStreamSerializationAllowed = 1;
    ++n;
  }
  cfg.attrs = attr;
  cfg.numAttrs = n;
  LCU_CUDA(cudaLaunchKernelEx(&cfg, kernel, static_cast<KP>(args)...));
  return LCU_OK;
}

}  // namespace lcu
