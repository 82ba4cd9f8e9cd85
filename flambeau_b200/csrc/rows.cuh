// What the row-wise kernels share: four elements at a time whatever the storage type, and elements of a row that is
// stored as several float32 shares.
#pragma once

#include "common.cuh"

template <typename T> struct Vec4 {};
template <> struct Vec4<float> {
    static __device__ __forceinline__ float4 load(const float* p) { return *reinterpret_cast<const float4*>(p); }
    static __device__ __forceinline__ void store(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
};
template <> struct Vec4<__nv_bfloat16> {
    static __device__ __forceinline__ float4 load(const __nv_bfloat16* p) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        return make_float4(a.x, a.y, b.x, b.y);
    }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, float4 v) {
        __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
        uint2 raw;
        raw.x = *reinterpret_cast<uint32_t*>(&a);
        raw.y = *reinterpret_cast<uint32_t*>(&b);
        *reinterpret_cast<uint2*>(p) = raw;
    }
};

// Element j of a row that is stored as `n_partials` slabs `partial_stride` elements apart (split-K shares).
template <typename TI>
__device__ __forceinline__ float slab_sum(const TI* __restrict__ row, int j, int n_partials, long partial_stride) {
    float acc = fb_to_float(row[j]);
    for (int p = 1; p < n_partials; p += 8) {         // eight independent loads in flight, added in slab order
        float a[8];
#pragma unroll
        for (int u = 0; u < 8; ++u)
            a[u] = p + u < n_partials ? fb_to_float(row[(size_t)(p + u) * partial_stride + j]) : 0.0f;
#pragma unroll
        for (int u = 0; u < 8; ++u) acc += a[u];
    }
    return acc;
}

template <typename TI>
__device__ __forceinline__ float4 slab_sum4(const TI* __restrict__ p, int n_partials, long partial_stride) {
    float4 acc = Vec4<TI>::load(p);
    for (int s = 1; s < n_partials; s += 8) {         // eight independent loads in flight, added in slab order
        float4 a[8];
#pragma unroll
        for (int u = 0; u < 8; ++u)
            a[u] = s + u < n_partials ? Vec4<TI>::load(p + (size_t)(s + u) * partial_stride) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int u = 0; u < 8; ++u) { acc.x += a[u].x; acc.y += a[u].y; acc.z += a[u].z; acc.w += a[u].w; }
    }
    return acc;
}
