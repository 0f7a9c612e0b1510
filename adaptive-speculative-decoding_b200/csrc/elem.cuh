// Element access for kernels that are instantiated for bf16 and for fp32 buffers, and block-wide sums.
#pragma once
#include <cuda_bf16.h>

namespace asd {

template <typename T>
__device__ __forceinline__ float ldf(const T* p) {
    return (float)*p;
}
template <>
__device__ __forceinline__ float ldf<__nv_bfloat16>(const __nv_bfloat16* p) {
    return __bfloat162float(*p);
}
template <typename T>
__device__ __forceinline__ void stf(T* p, float v) {
    *p = v;
}
template <>
__device__ __forceinline__ void stf<__nv_bfloat16>(__nv_bfloat16* p, float v) {
    *p = __float2bfloat16(v);
}
// runtime-typed forms (f32 flag: 0 = bf16, 1 = fp32) for kernels whose arithmetic dwarfs the branch
__device__ __forceinline__ float ldx(const void* p, long long i, int f32) {
    return f32 ? ((const float*)p)[i] : __bfloat162float(((const __nv_bfloat16*)p)[i]);
}
// four consecutive elements from a place that is a multiple of four in a 16-byte aligned buffer
__device__ __forceinline__ void ldx4(const void* p, long long i, int f32, float (&v)[4]) {
    if (f32) {
        const float4 f = *reinterpret_cast<const float4*>((const float*)p + i);
        v[0] = f.x, v[1] = f.y, v[2] = f.z, v[3] = f.w;
    } else {
        const uint2 r = *reinterpret_cast<const uint2*>((const __nv_bfloat16*)p + i);
        v[0] = __uint_as_float(r.x << 16), v[1] = __uint_as_float(r.x & 0xffff0000u);
        v[2] = __uint_as_float(r.y << 16), v[3] = __uint_as_float(r.y & 0xffff0000u);
    }
}
__device__ __forceinline__ void stx(void* p, long long i, int f32, float v) {
    if (f32)
        ((float*)p)[i] = v;
    else
        ((__nv_bfloat16*)p)[i] = __float2bfloat16(v);
}
// four consecutive elements to a place that is a multiple of four in a 16-byte aligned buffer
__device__ __forceinline__ void stx4(void* p, long long i, int f32, const float (&v)[4]) {
    if (f32) {
        *reinterpret_cast<float4*>((float*)p + i) = make_float4(v[0], v[1], v[2], v[3]);
    } else {
        __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>((__nv_bfloat16*)p + i) =
            make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
    }
}

// two fp32 operations in one instruction (each rounded as its scalar form)
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
    unsigned long long d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;"
        : "=l"(d)
        : "l"(*reinterpret_cast<unsigned long long*>(&a)), "l"(*reinterpret_cast<unsigned long long*>(&b)),
          "l"(*reinterpret_cast<unsigned long long*>(&c)));
    return *reinterpret_cast<float2*>(&d);
}
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
    unsigned long long d;
    asm("mul.rn.f32x2 %0, %1, %2;"
        : "=l"(d)
        : "l"(*reinterpret_cast<unsigned long long*>(&a)), "l"(*reinterpret_cast<unsigned long long*>(&b)));
    return *reinterpret_cast<float2*>(&d);
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
// sum over the block in a fixed order (warp sums, then the warps in index order); red: >= 33 floats of shared memory
__device__ __forceinline__ float block_sum(float v, float* red) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
    v = warp_sum(v);
    __syncthreads();
    if (lane == 0) red[warp] = v;
    __syncthreads();
    if (threadIdx.x == 0) {
        float t = 0.f;
        for (int i = 0; i < nw; ++i) t += red[i];
        red[32] = t;
    }
    __syncthreads();
    return red[32];
}

}  // namespace asd
