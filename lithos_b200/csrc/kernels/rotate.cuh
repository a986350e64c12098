// Cache elements (bf16 or fp32) and rotations of neighbouring pairs by position, shared by the attention kernels of list-of-layers models.
#pragma once
#include "common.cuh"
#include "params.h"

template <typename T> struct wa_t;
template <> struct wa_t<__nv_bfloat16> {
    static __device__ __forceinline__ void ld8(const __nv_bfloat16* p, float (&f)[8]) {
        const uint4 u = *reinterpret_cast<const uint4*>(p);
        const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            f[2 * i] = __uint_as_float(w[i] << 16);
            f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
        }
    }
    static __device__ __forceinline__ float2 ld2(const __nv_bfloat16* p) {
        const uint32_t u = *reinterpret_cast<const uint32_t*>(p);
        return make_float2(__uint_as_float(u << 16), __uint_as_float(u & 0xffff0000u));
    }
    static __device__ __forceinline__ __nv_bfloat16 from(float v) { return __float2bfloat16_rn(v); }
};
template <> struct wa_t<float> {
    static __device__ __forceinline__ void ld8(const float* p, float (&f)[8]) {
        const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
        f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
    }
    static __device__ __forceinline__ float2 ld2(const float* p) { return *reinterpret_cast<const float2*>(p); }
    static __device__ __forceinline__ float from(float v) { return v; }
};

__device__ __forceinline__ void wa_angle(double f, int pos, float& c, float& s) { // product and reduction modulo 2 pi in double
    const double a = (double)pos * f, k = rint(a * 0.15915494309189535);
    sincosf((float)fma(-k, 6.283185307179586, a), &s, &c);
}
// one warp: dst[0..dim) = rotated src (times mul)
template <typename T>
__device__ __forceinline__ void wa_warp_rotate(const float* src, T* dst, int dim, int rot_dims, const float* cs, const float* sn, float mul) {
    for (int i = threadIdx.x & 31; i < (dim + 1) / 2; i += 32) {
        float u = src[2 * i], v = 2 * i + 1 < dim ? src[2 * i + 1] : 0.f;
        if (2 * i < rot_dims) {
            const float a = u * cs[i] - v * sn[i];
            v = v * cs[i] + u * sn[i];
            u = a;
        }
        dst[2 * i] = wa_t<T>::from(u * mul);
        if (2 * i + 1 < dim) dst[2 * i + 1] = wa_t<T>::from(v * mul);
    }
}
