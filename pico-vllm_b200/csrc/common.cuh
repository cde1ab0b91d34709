// Shared helpers of the kernels: element types, conversions, warp and block reductions.
#pragma once
#include <cuda_runtime.h>
#include <cuda_bf16.h>
#include <stdint.h>
#include <math.h>

#define PICO_API extern "C" __attribute__((visibility("default")))

// error codes returned by the host entry points (0 = launched; >0 = cudaError_t of the launch)
#define PICO_ERR_DTYPE (-2)
#define PICO_ERR_SIZE (-3)
#define PICO_ERR_ALIGN (-4)

enum PicoDType { PICO_F32 = 0, PICO_BF16 = 1 };

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

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

// Sum over the whole block; every thread gets the result.  scratch: 33 floats of shared memory.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int nwarps = (blockDim.x + 31) >> 5;
    v = warp_sum(v);
    __syncthreads();  // scratch may still be read from an earlier call
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    if (warp == 0) {
        float t = lane < nwarps ? scratch[lane] : 0.f;
        t = warp_sum(t);
        if (lane == 0) scratch[32] = t;
    }
    __syncthreads();
    return scratch[32];
}
__device__ __forceinline__ float block_max(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int nwarps = (blockDim.x + 31) >> 5;
    v = warp_max(v);
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    if (warp == 0) {
        float t = lane < nwarps ? scratch[lane] : -INFINITY;
        t = warp_max(t);
        if (lane == 0) scratch[32] = t;
    }
    __syncthreads();
    return scratch[32];
}

// An attention score in log2 units (the softmax uses exp2): raw * scale_log2, or, with a soft cap c on the scaled score,
// c * tanh(raw * scale / c) in the same units.  cap_log2 = c * log2(e) (0: no cap); cap_2x = 2 * scale / c.
// tanh(x) = 1 - 2 / (e^(2x) + 1): exact at both ends, absolute error ~1e-7 near 0.
__device__ __forceinline__ float pico_score_log2(float raw, float scale_log2, float cap_log2, float cap_2x) {
    if (cap_log2 > 0.f) return cap_log2 * (1.0f - __fdividef(2.0f, __expf(raw * cap_2x) + 1.0f));
    return raw * scale_log2;
}

// What a distance bias takes off a score, in log2 units.  Linear: slope2 * distance with slope2 = slope * log2(e).  With a
// rate: slope * ln(1 + rate * distance) * log2(e) = slope * log2(1 + rate * distance).
__device__ __forceinline__ float pico_log_bias(float slope, float rate, float distance) {
    return slope * __log2f(fmaxf(fmaf(rate, distance, 1.0f), 1e-30f));
}

static inline int pico_launch_status() { return (int)cudaGetLastError(); }

// Multiprocessors of the current device (asked once per device; grids are sized from it).
static inline int pico_num_sms() {
    static int cached[64] = {0};
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) dev = 0;
    if (cached[dev] <= 0) {
        int sms = 0;
        if (cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || sms <= 0) sms = 1;
        cached[dev] = sms;
    }
    return cached[dev];
}

// Programmatic dependent launch: every kernel of this library is launched with the attribute that
// lets it start while the kernel before it in the stream is still draining, and therefore begins
// with pdl_launch_dependents() (the next kernel may be scheduled) and calls pdl_wait() before it
// touches anything an earlier kernel wrote (pdl_wait returns when the earlier grids have completed
// and their writes are visible).  What a kernel does before pdl_wait - setting up barriers,
// prefetching weights - overlaps the earlier kernel's tail.
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;\n" ::: "memory"); }
__device__ __forceinline__ void pdl_launch_dependents() { asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory"); }

// cluster_x > 1: the blocks of grid.x are launched as thread-block clusters of that many blocks.
template <typename... KArgs, typename... Args>
static inline void pico_launch_cluster(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem,
                                       cudaStream_t stream, int cluster_x, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    int n = 1;
    if (cluster_x > 1) {
        attr[1].id = cudaLaunchAttributeClusterDimension;
        attr[1].val.clusterDim.x = cluster_x;
        attr[1].val.clusterDim.y = 1;
        attr[1].val.clusterDim.z = 1;
        n = 2;
    }
    cfg.attrs = attr;
    cfg.numAttrs = n;
    cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...);
}

template <typename... KArgs, typename... Args>
static inline void pico_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                               Args... args) {
    pico_launch_cluster(kernel, grid, block, smem, stream, 1, args...);
}
