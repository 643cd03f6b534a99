// Shared pieces of the layer-list model kernels (dense.cu, norms.cu, latent_attention.cu, mamba2.cu):
// element types of weights and caches, exact roundings, launch checking.
//
// These kernels keep every activation that crosses a kernel boundary in f32.  Weights are bf16 or f32
// ("wtype"), caches bf16 or f32 ("ctype"); a matrix product in bf16 mode rounds its activation operand to
// bf16 on the way in and accumulates in f32, exactly what a bf16 tensor-core product does.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#define DL_T_F32 0
#define DL_T_BF16 1

extern void dl_set_error(const char* fmt, ...);

#define LAYER_CHECK_LAUNCH(name)                                                        \
    do {                                                                                \
        cudaError_t e__ = cudaGetLastError();                                           \
        if (e__ != cudaSuccess) {                                                       \
            dl_set_error("%s: %s", name, cudaGetErrorString(e__));                      \
            return -(int)e__;                                                           \
        }                                                                               \
    } while (0)

template <typename T> __device__ __forceinline__ float ld_f(const T* p);
template <> __device__ __forceinline__ float ld_f<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ld_f<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }

template <typename T> __device__ __forceinline__ void st_f(T* p, float v);
template <> __device__ __forceinline__ void st_f<float>(float* p, float v) { *p = v; }
template <> __device__ __forceinline__ void st_f<__nv_bfloat16>(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

__device__ __forceinline__ float round_bf16(float v) { return __bfloat162float(__float2bfloat16_rn(v)); }

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

// sum over the block; `red` is >= 32 floats of shared memory; every thread gets the result
__device__ __forceinline__ float block_sum(float v, float* red) {
    v = warp_sum(v);
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = (blockDim.x + 31) >> 5;
    __syncthreads();
    if (l == 0) red[w] = v;
    __syncthreads();
    float t = (l < nw) ? red[l] : 0.f;
    t = warp_sum(t);
    return t;
}

__device__ __forceinline__ float silu_f(float v) { return v / (1.f + expf(-v)); }
__device__ __forceinline__ float sigmoid_f(float v) { return 1.f / (1.f + expf(-v)); }
__device__ __forceinline__ float softplus_f(float v) { return v > 20.f ? v : log1pf(expf(v)); }

// sigma(v) and 1 - sigma(v), both without cancellation.  The divisor lies in [1, 2], where the fast division is good to 2 ulp (and
// brings no slow-path call into kernels that hold much in registers)
__device__ __forceinline__ void sigmoid_pair_f(float v, float& s, float& c) {
    const float e = expf(-fabsf(v)), r = __fdividef(1.f, 1.f + e);
    s = v >= 0.f ? r : e * r;
    c = v >= 0.f ? e * r : r;
}
__device__ __forceinline__ float gelu_tanh_f(float v) {
    return 0.5f * v * (1.f + tanhf(0.7978845608028654f * fmaf(0.044715f * v * v, v, v)));
}

// Activation image of the tcgen05 GEMM (see dense.cu): bytes from the image's start to element (row m, column k).  Eight
// neighbouring columns k .. k + 7 (k % 8 == 0) of a row are 16 consecutive bytes.
__device__ __forceinline__ size_t xh_offset(int ncap, int m, int k) {
    return ((size_t)(k >> 7) * (ncap >> 3) + (m >> 3)) * 2048 + (size_t)((k & 127) >> 3) * 128 + (m & 7) * 16 + (k & 7) * 2;
}
__device__ __forceinline__ void xh_store(uint8_t* xh, int ncap, int m, int k, float v) {
    *reinterpret_cast<__nv_bfloat16*>(xh + xh_offset(ncap, m, k)) = __float2bfloat16_rn(v);
}
// zeros in columns [K, round_up(K, 128)) of row m, by the threads of one CTA or warp (thread t of n)
__device__ __forceinline__ void xh_zero_tail(uint8_t* xh, int ncap, int m, int K, int t, int n) {
    for (int k = K + t; k < ((K + 127) & ~127); k += n) xh_store(xh, ncap, m, k, 0.f);
}
