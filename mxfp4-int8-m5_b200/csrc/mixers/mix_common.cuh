// Shared helpers of the sequence-mixer kernels: activation storage types (bfloat16 bits or float), float reductions,
// activation functions in 32-bit, and the rotate-half table.
#pragma once
#include "../scmx_common.cuh"
#include "../../../include/scmx_mixers.h"

namespace scmx {

typedef uint16_t bf16_t;      // storage type of a bfloat16 value

__device__ __forceinline__ float ldf(const bf16_t* p) { return bf16_to_f32(*p); }
__device__ __forceinline__ float ldf(const float* p) { return *p; }
__device__ __forceinline__ void stf(bf16_t* p, float v) { *p = f32_to_bf16(v); }
__device__ __forceinline__ void stf(float* p, float v) { *p = v; }

// Eight consecutive values (16-byte aligned for bf16, 16-byte aligned halves for float).
__device__ __forceinline__ void ld8(const bf16_t* p, float (&v)[8]) {
    const uint4 w = *reinterpret_cast<const uint4*>(p);
    const uint32_t u[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        v[2 * i] = bf16_lo(u[i]);
        v[2 * i + 1] = bf16_hi(u[i]);
    }
}
__device__ __forceinline__ void ld8(const float* p, float (&v)[8]) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
// Eight stored values as loaded, converted on use.
template <typename T> struct Raw8;
template <> struct Raw8<bf16_t> {
    uint4 w;
    __device__ __forceinline__ void load(const bf16_t* p) { w = *reinterpret_cast<const uint4*>(p); }
    __device__ __forceinline__ void store(bf16_t* p) const { *reinterpret_cast<uint4*>(p) = w; }
    __device__ __forceinline__ void get(float (&x)[8]) const {
        x[0] = bf16_lo(w.x); x[1] = bf16_hi(w.x); x[2] = bf16_lo(w.y); x[3] = bf16_hi(w.y);
        x[4] = bf16_lo(w.z); x[5] = bf16_hi(w.z); x[6] = bf16_lo(w.w); x[7] = bf16_hi(w.w);
    }
};
template <> struct Raw8<float> {
    float4 a, b;
    __device__ __forceinline__ void load(const float* p) { a = reinterpret_cast<const float4*>(p)[0]; b = reinterpret_cast<const float4*>(p)[1]; }
    __device__ __forceinline__ void store(float* p) const {
        reinterpret_cast<float4*>(p)[0] = a;
        reinterpret_cast<float4*>(p)[1] = b;
    }
    __device__ __forceinline__ void get(float (&x)[8]) const {
        x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w; x[4] = b.x; x[5] = b.y; x[6] = b.z; x[7] = b.w;
    }
};

// Four consecutive values.
__device__ __forceinline__ void st4(bf16_t* p, float a, float b, float c, float d) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(a, b), pack_bf16x2(c, d));
}
__device__ __forceinline__ void st4(float* p, float a, float b, float c, float d) {
    *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
}
__device__ __forceinline__ float4 ld4(const bf16_t* p) {
    const uint2 w = *reinterpret_cast<const uint2*>(p);
    return make_float4(bf16_lo(w.x), bf16_hi(w.x), bf16_lo(w.y), bf16_hi(w.y));
}
__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }

__device__ __forceinline__ float warp_sumf(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// Block-wide sum; `red` holds 33 floats; every thread gets the result.
__device__ __forceinline__ float block_sumf(float v, float* red) {
    const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, nw = blockDim.x >> 5;
    v = warp_sumf(v);
    __syncthreads();
    if (lane == 0) red[w] = v;
    __syncthreads();
    if (w == 0) {
        const float t = warp_sumf(lane < nw ? red[lane] : 0.0f);
        if (lane == 0) red[32] = t;
    }
    __syncthreads();
    return red[32];
}

// Packed float32 pairs.
__device__ __forceinline__ uint64_t pack2(float lo, float hi) {
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ float2 unpack2(uint64_t v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
    uint64_t r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}

__device__ __forceinline__ float rms_inv_f32(float sumsq, int n, float eps) { return 1.0f / sqrtf(sumsq / (float)n + eps); }
// 2^x by the special-function unit, results below the normal range flushed to zero.
__device__ __forceinline__ float ex2_approx(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float exp_fast(float z) { return ex2_approx(z * 1.4426950408889634f); }
__device__ __forceinline__ float silu_f32(float z) { return __fdividef(z, 1.0f + exp_fast(-z)); }
// log(1 + e^z) = max(z, 0) + log(1 + e), e = e^-|z| in (0, 1]; log(1 + e) / e as the polynomial that interpolates it in the ten
// Chebyshev points of [0, 1] (relative error below 2e-7, so small steps keep their precision).
__device__ __forceinline__ float softplus_f32(float z) {
    const float e = exp_fast(-fabsf(z));
    float p = -3.176057013e-03f;
    p = fmaf(p, e, 1.954252832e-02f);
    p = fmaf(p, e, -5.637361482e-02f);
    p = fmaf(p, e, 1.054362357e-01f);
    p = fmaf(p, e, -1.526966691e-01f);
    p = fmaf(p, e, 1.966327429e-01f);
    p = fmaf(p, e, -2.495161593e-01f);
    p = fmaf(p, e, 3.332971036e-01f);
    p = fmaf(p, e, -4.999989271e-01f);
    p = fmaf(p, e, 1.0f);
    return fmaf(p, e, fmaxf(z, 0.0f));
}
// xIELU with a_pos = softplus(p) and a_neg = 1/2 + softplus(q): quadratic above zero, exponential below, slope 1/2 at zero.
// e^z - 1 - z near zero by its Taylor series (seven terms: relative error 5e-8 on [-1/2, 0]), where the difference would cancel.
__device__ __forceinline__ float xielu_f32(float z, float a_pos, float a_neg) {
    float s = 1.0f / 40320.0f;
    s = fmaf(s, z, 1.0f / 5040.0f);
    s = fmaf(s, z, 1.0f / 720.0f);
    s = fmaf(s, z, 1.0f / 120.0f);
    s = fmaf(s, z, 1.0f / 24.0f);
    s = fmaf(s, z, 1.0f / 6.0f);
    s = fmaf(s, z, 0.5f);
    const float far = exp_fast(z) - 1.0f - z;
    const float neg = z > -0.5f ? s * z * z : far;
    return fmaf(0.5f, z, z > 0.0f ? a_pos * z * z : a_neg * neg);
}

__device__ __forceinline__ float sigmoid_f32(float z) { return __fdividef(1.0f, 1.0f + exp_fast(-z)); }
// z / 2 (1 + tanh(u)) = z sigmoid(2 u), u = sqrt(2 / pi) (z + 0.044715 z^3).
__device__ __forceinline__ float gelu_tanh_f32(float z) {
    const float u = 0.7978845608028654f * fmaf(0.044715f * z * z, z, z);
    return z * sigmoid_f32(2.0f * u);
}

// Element i of a head vector of size d after the rotate-half rotation of its first `dims` elements: i < dims/2 pairs with
// i + dims/2.  cs: the position's table row, cos (dims/2) then sin (dims/2).
template <typename T>
__device__ __forceinline__ float rotated(const T* v, int i, int dims, const float* cs) {
    const float self = ldf(v + i);
    if (i >= dims) return self;
    const int half = dims >> 1;
    if (i < half) return self * cs[i] - ldf(v + i + half) * cs[half + i];
    return self * cs[i - half] + ldf(v + i - half) * cs[i];
}

#define SCMX_DT_OK(who, dt) SCMX_REQUIRE((dt) == 0 || (dt) == 1, SCMX_EINVAL, "%s: dtype %d (0 = bfloat16, 1 = float)", who, dt)

}  // namespace scmx
