// Device helpers of the row-count kernels: bf16 <-> fp32, element access by activation type, warp-group sums.
#pragma once
#include <cuda_bf16.h>
#include "common.cuh"

namespace gehtp {

__device__ __forceinline__ float bf2f(uint16_t h) { return __uint_as_float((uint32_t)h << 16); }
__device__ __forceinline__ uint16_t f2bf(float f) { return __bfloat16_as_ushort(__float2bfloat16_rn(f)); }
__device__ __forceinline__ uint32_t pack_bf2(float lo, float hi) {
    const __nv_bfloat162 p = __floats2bfloat162_rn(lo, hi);
    return *(const uint32_t*)&p;
}

// activation element types
struct ActF32 {
    typedef float T;
    static __device__ __forceinline__ float ld(const float* p) { return __ldcg(p); }
    static __device__ __forceinline__ void st(float* p, float v) { *p = v; }
};
struct ActBf16 {
    typedef uint16_t T;
    static __device__ __forceinline__ float ld(const uint16_t* p) { return bf2f(__ldcg(p)); }
    static __device__ __forceinline__ void st(uint16_t* p, float v) { *p = f2bf(v); }
};

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
// the same on the hardware exponential and reciprocal, within a few 2^-23 of it: beside outputs that are rounded to bf16
__device__ __forceinline__ float sigmoid_fast(float z) { return __fdividef(1.0f, 1.0f + __expf(fminf(-z, 80.0f))); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }

// sum over the whole block; `part` holds one float per warp. Every thread gets the sum.
__device__ __forceinline__ float block_sum(float v, float* part) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = (blockDim.x + 31) >> 5;
    v = warp_sum(v);
    __syncthreads();
    if (lane == 0) part[warp] = v;
    __syncthreads();
    float s = 0.0f;
    for (int w = 0; w < nw; w++) s += part[w];
    return s;
}

// Cluster barrier in two halves: all threads of the cluster's CTAs arrive, then wait.
__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }

__device__ __forceinline__ void pdl_release() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }

}  // namespace gehtp
