// Loads, stores and elementwise functions over 1, 4 or 8 consecutive elements of bf16 or fp32 activations.
#pragma once

#include "nckv_common.cuh"

namespace nckv {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float *p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16 *p, float v) { *p = __float2bfloat16_rn(v); }

// V consecutive elements
__device__ __forceinline__ void get_v(const float *p, float (&o)[1]) { o[0] = p[0]; }
__device__ __forceinline__ void get_v(const __nv_bfloat16 *p, float (&o)[1]) { o[0] = to_f(p[0]); }
__device__ __forceinline__ void get_v(const float *p, float (&o)[4]) {
    const float4 f = *reinterpret_cast<const float4 *>(p);
    o[0] = f.x; o[1] = f.y; o[2] = f.z; o[3] = f.w;
}
__device__ __forceinline__ void get_v(const __nv_bfloat16 *p, float (&o)[4]) {
    const uint2 f = *reinterpret_cast<const uint2 *>(p);
    o[0] = bf16lo(f.x); o[1] = bf16hi(f.x); o[2] = bf16lo(f.y); o[3] = bf16hi(f.y);
}
__device__ __forceinline__ void put_v(float *p, const float (&o)[1]) { p[0] = o[0]; }
__device__ __forceinline__ void put_v(__nv_bfloat16 *p, const float (&o)[1]) { put(p, o[0]); }
__device__ __forceinline__ void put_v(float *p, const float (&o)[4]) {
    *reinterpret_cast<float4 *>(p) = make_float4(o[0], o[1], o[2], o[3]);
}
__device__ __forceinline__ void put_v(__nv_bfloat16 *p, const float (&o)[4]) {
    *reinterpret_cast<uint2 *>(p) = make_uint2(pack_bf16x2(o[0], o[1]), pack_bf16x2(o[2], o[3]));
}

__device__ __forceinline__ void get_v(const float *p, float (&o)[8]) {
    const float4 a = reinterpret_cast<const float4 *>(p)[0], b = reinterpret_cast<const float4 *>(p)[1];
    o[0] = a.x; o[1] = a.y; o[2] = a.z; o[3] = a.w; o[4] = b.x; o[5] = b.y; o[6] = b.z; o[7] = b.w;
}
__device__ __forceinline__ void get_v(const __nv_bfloat16 *p, float (&o)[8]) {
    const uint4 f = *reinterpret_cast<const uint4 *>(p);
    o[0] = bf16lo(f.x); o[1] = bf16hi(f.x); o[2] = bf16lo(f.y); o[3] = bf16hi(f.y);
    o[4] = bf16lo(f.z); o[5] = bf16hi(f.z); o[6] = bf16lo(f.w); o[7] = bf16hi(f.w);
}
__device__ __forceinline__ void put_v(float *p, const float (&o)[8]) {
    reinterpret_cast<float4 *>(p)[0] = make_float4(o[0], o[1], o[2], o[3]);
    reinterpret_cast<float4 *>(p)[1] = make_float4(o[4], o[5], o[6], o[7]);
}
__device__ __forceinline__ void put_v(__nv_bfloat16 *p, const float (&o)[8]) {
    *reinterpret_cast<uint4 *>(p) = make_uint4(pack_bf16x2(o[0], o[1]), pack_bf16x2(o[2], o[3]), pack_bf16x2(o[4], o[5]), pack_bf16x2(o[6], o[7]));
}

// Elementwise functions in fp32: bf16 activations get the fast intrinsics (a few fp32 ulps, tanh aside), fp32 ones
// the full-precision functions.
template <typename T> struct Fn;
template <> struct Fn<float> {
    static __device__ __forceinline__ float exp(float x) { return expf(x); }
    static __device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
    static __device__ __forceinline__ float silu(float z) { return z / (1.f + expf(-z)); }
    static __device__ __forceinline__ float tanh(float z) { return tanhf(z); }
};
template <> struct Fn<__nv_bfloat16> {
    static __device__ __forceinline__ float exp(float x) { return __expf(x); }
    static __device__ __forceinline__ float sigmoid(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }
    static __device__ __forceinline__ float silu(float z) { return __fdividef(z, 1.f + __expf(-z)); }
    static __device__ __forceinline__ float tanh(float z) {  // 11 bits, more than a bf16 activation holds
        float r;
        asm("tanh.approx.f32 %0, %1;" : "=f"(r) : "f"(z));
        return r;
    }
};
// log(1 + e^z) without overflow
__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
template <typename T> __device__ __forceinline__ float gelu_tanh(float z) {
    return 0.5f * z * (1.f + Fn<T>::tanh(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

}  // namespace nckv
