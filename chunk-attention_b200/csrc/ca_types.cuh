// Element types of the device code: conversion to and from fp32 and small vector accesses, for fp32, fp16 and bf16.
#pragma once
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <stdint.h>

namespace ca {

__device__ __forceinline__ float to_f32(float x) { return x; }
__device__ __forceinline__ float to_f32(__half x) { return __half2float(x); }
__device__ __forceinline__ float to_f32(__nv_bfloat16 x) { return __bfloat162float(x); }

template <typename T> __device__ __forceinline__ T from_f32(float x);
template <> __device__ __forceinline__ float from_f32<float>(float x) { return x; }
template <> __device__ __forceinline__ __half from_f32<__half>(float x) { return __float2half_rn(x); }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float x) { return __float2bfloat16_rn(x); }

template <typename T, int N> struct alignas(sizeof(T) * N) Pack { T v[N]; };

// one 16-byte granule of T as floats
template <typename T> struct Granule {
    static constexpr int N = 16 / sizeof(T);
    static __device__ __forceinline__ void load(const T* p, float* out) {
        const Pack<T, N> x = *reinterpret_cast<const Pack<T, N>*>(p);
#pragma unroll
        for (int i = 0; i < N; i++) out[i] = to_f32(x.v[i]);
    }
};

__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int off = 16; off >= 1; off >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, off));
    return v;
}
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int off = 16; off >= 1; off >>= 1) v += __shfl_xor_sync(0xffffffffu, v, off);
    return v;
}

// sine and cosine for 16-bit kernels: the angle is brought into [-pi, pi] in two fp32 steps, then the hardware
// functions (absolute error below 2^-20)
__device__ __forceinline__ void fast_sincos(float a, float* sn, float* cs) {
    const float k = rintf(a * 0.15915494309189535f);
    float r = fmaf(k, -6.2831854820251465f, a);   // 2 pi rounded to fp32 ...
    r = fmaf(k, 1.7484556e-7f, r);                // ... and what the rounding added
    *sn = __sinf(r);
    *cs = __cosf(r);
}
template <typename T> __device__ __forceinline__ void sincos_for(float a, float* sn, float* cs) { fast_sincos(a, sn, cs); }
template <> __device__ __forceinline__ void sincos_for<float>(float a, float* sn, float* cs) { sincosf(a, sn, cs); }

// sine and cosine of pos * f, f = hi + lo.  fp32 kernels keep what the product's rounding and hi leave out; in 16-bit kernels
// it is far below the results' own rounding.
template <typename T> __device__ __forceinline__ void turn_for(float pos, float hi, float lo, float* sn, float* cs) { fast_sincos(pos * hi, sn, cs); }
template <> __device__ __forceinline__ void turn_for<float>(float pos, float hi, float lo, float* sn, float* cs) {
    const float a = pos * hi, rest = fmaf(pos, lo, fmaf(pos, hi, -a));
    float s, c;
    sincosf(a, &s, &c);
    *sn = fmaf(rest, c, s);
    *cs = fmaf(-rest, s, c);
}

// one MUFU operation; results below 2^-126 are 0
__device__ __forceinline__ float exp2_approx(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float rcp_approx(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// pairs of fp32 in one 64-bit register: two results per instruction, each rounded as the scalar one
__device__ __forceinline__ uint64_t pair_f32(float lo, float hi) {
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ void unpair_f32(uint64_t v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ uint64_t mul_f32x2(uint64_t a, uint64_t b) {
    uint64_t r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ uint64_t fma_f32x2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
// for results that are rounded to T: kernels of 16-bit types use the hardware approximations (relative error about 2^-21)
template <typename T> __device__ __forceinline__ float sigmoid_for(float z) { return rcp_approx(1.f + exp2_approx(-1.4426950408889634f * z)); }
template <> __device__ __forceinline__ float sigmoid_for<float>(float z) { return sigmoid_f(z); }
template <typename T> __device__ __forceinline__ float silu_for(float z) { return z * sigmoid_for<T>(z); }
template <> __device__ __forceinline__ float silu_for<float>(float z) { return silu_f(z); }

// log(1 + exp(z)) = max(z, 0) + log(1 + e), e = exp(-|z|) in (0, 1], with log(1 + e) = 2 artanh(s), s = e / (2 + e) <= 1/3,
// by its power series up to s^13 (the rest is below 2^-25 of the sum)
__device__ __forceinline__ float softplus_f(float z) {
    const float e = exp2f(-1.4426950408889634f * fabsf(z));
    const float s = __fdividef(e, 2.f + e), q = s * s;
    float a = fmaf(q, 1.f / 13.f, 1.f / 11.f);
    a = fmaf(q, a, 1.f / 9.f);
    a = fmaf(q, a, 1.f / 7.f);
    a = fmaf(q, a, 1.f / 5.f);
    a = fmaf(q, a, 1.f / 3.f);
    a = fmaf(q, a, 1.f);
    return fmaf(2.f * s, a, fmaxf(z, 0.f));
}

}  // namespace ca
