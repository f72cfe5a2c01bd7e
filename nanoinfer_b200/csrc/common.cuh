// Shared device helpers of the sm_100a kernels.  Header only; every .cu file of this
// folder is built into a shared library of its own and exports plain C functions that
// take device pointers and a stream and return 0 or an error code.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#define NI_DTYPE_F32 0
#define NI_DTYPE_BF16 1

// Error codes of the exported functions: positive = a cudaError_t, negative = ours.
#define NI_OK 0
#define NI_ERR_BAD_ARGUMENT (-1)
#define NI_ERR_UNSUPPORTED_SIZE (-2)
#define NI_ERR_DEVICE_TIMEOUT (-3)

#define NI_EXPORT extern "C" __attribute__((visibility("default")))

#define NI_RETURN_LAUNCH_STATUS()                      \
    do {                                               \
        cudaError_t e__ = cudaGetLastError();          \
        return e__ == cudaSuccess ? NI_OK : (int)e__;  \
    } while (0)

// Streaming multiprocessors of the current device (asked once per device; 148 on a B200).
// Grid sizes and work splits are derived from it, never from a literal.
static inline int ni_sm_count() {
    static int cached[64];
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) dev = 0;
    if (cached[dev] <= 0) {
        int n = 0;
        if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || n <= 0) n = 1;
        cached[dev] = n;
    }
    return cached[dev];
}

template <typename T> __device__ __forceinline__ float ni_to_float(T v);
template <> __device__ __forceinline__ float ni_to_float<float>(float v) { return v; }
template <> __device__ __forceinline__ float ni_to_float<__nv_bfloat16>(__nv_bfloat16 v) {
    return __bfloat162float(v);
}
template <typename T> __device__ __forceinline__ T ni_from_float(float v);
template <> __device__ __forceinline__ float ni_from_float<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 ni_from_float<__nv_bfloat16>(float v) {
    return __float2bfloat16_rn(v);
}

__device__ __forceinline__ float ni_warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float ni_warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// Sum over a block of up to 1024 threads, same value in every thread, fixed order.
// `scratch` holds 32 floats of shared memory.
__device__ __forceinline__ float ni_block_sum(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int nwarps = (blockDim.x + 31) >> 5;
    v = ni_warp_sum(v);
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    float t = 0.f;
    for (int w = 0; w < nwarps; ++w) t += scratch[w];
    return t;
}
__device__ __forceinline__ float ni_block_max(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int nwarps = (blockDim.x + 31) >> 5;
    v = ni_warp_max(v);
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    float t = scratch[0];
    for (int w = 1; w < nwarps; ++w) t = fmaxf(t, scratch[w]);
    return t;
}

// Activation of a gated unit's gate: g * sigmoid(g (c1 + c2 g^2)).  (1, 0) is silu; (2 sqrt(2 / pi), 0.044715 of that) is the
// tanh form of gelu, since (1 + tanh y) / 2 = sigmoid(2 y).
#define NI_GELU_C1 1.5957691216057308f
#define NI_GELU_C2 0.07135481627159896f
__device__ __forceinline__ float ni_gate_act(float g, float c1, float c2) {
    return g / (1.0f + expf(-(g * fmaf(c2 * g, g, c1))));
}
// The mode of a product with a gated epilogue may carry this flag: gelu instead of silu.
#define NI_MODE_GELU 16

// 16 bytes of a row at once: 8 bfloat16 or 4 float values, widened to FP32 (the address must be 16-byte aligned).
template <typename T> struct NiVec16;
template <> struct NiVec16<float> {
    static constexpr int N = 4;
    static __device__ __forceinline__ void load(const float* p, float* v) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
    }
    static __device__ __forceinline__ void store(float* p, const float* v) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    }
};
template <> struct NiVec16<__nv_bfloat16> {
    static constexpr int N = 8;
    static __device__ __forceinline__ void load(const __nv_bfloat16* p, float* v) {
        const uint4 x = *reinterpret_cast<const uint4*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&x);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float2 f = __bfloat1622float2(h[i]);
            v[2 * i] = f.x;
            v[2 * i + 1] = f.y;
        }
    }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, const float* v) {
        uint4 x;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&x);
#pragma unroll
        for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
        *reinterpret_cast<uint4*>(p) = x;
    }
};
