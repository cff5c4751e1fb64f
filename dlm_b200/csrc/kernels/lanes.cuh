// V (1, 2 or 4) neighbouring elements of a row as 32-bit values: loads and stores of float and bfloat16 rows in one access
// (the address must be a multiple of the access's size).
#pragma once
#include <cuda_bf16.h>

#include <cstdint>

namespace dlmk {

template <int V> struct Lanes { float v[V]; };
template <int V> __device__ __forceinline__ Lanes<V> load_f32(const float* p) {
    Lanes<V> r;
    if constexpr (V == 4) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        r.v[0] = x.x; r.v[1] = x.y; r.v[2] = x.z; r.v[3] = x.w;
    } else if constexpr (V == 2) {
        const float2 x = *reinterpret_cast<const float2*>(p);
        r.v[0] = x.x; r.v[1] = x.y;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <int V> __device__ __forceinline__ Lanes<V> load_act(const float* p) { return load_f32<V>(p); }
template <int V> __device__ __forceinline__ Lanes<V> load_act(const __nv_bfloat16* p) {
    Lanes<V> r;
    if constexpr (V == 1) {
        r.v[0] = __bfloat162float(*p);
    } else {
        uint32_t w[V / 2];
        if constexpr (V == 4) {
            const uint2 x = *reinterpret_cast<const uint2*>(p);
            w[0] = x.x; w[1] = x.y;
        } else {
            w[0] = *reinterpret_cast<const uint32_t*>(p);
        }
#pragma unroll
        for (int i = 0; i < V / 2; ++i) {
            r.v[2 * i] = __uint_as_float(w[i] << 16);
            r.v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
        }
    }
    return r;
}
template <int V> __device__ __forceinline__ void store_act(float* p, const Lanes<V>& r) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else if constexpr (V == 2) *reinterpret_cast<float2*>(p) = make_float2(r.v[0], r.v[1]);
    else *p = r.v[0];
}
template <int V> __device__ __forceinline__ void store_act(__nv_bfloat16* p, const Lanes<V>& r) {
    if constexpr (V == 1) {
        *p = __float2bfloat16_rn(r.v[0]);
    } else {
        uint32_t w[V / 2];
#pragma unroll
        for (int i = 0; i < V / 2; ++i) {
            const __nv_bfloat162 b = __floats2bfloat162_rn(r.v[2 * i], r.v[2 * i + 1]);
            w[i] = *reinterpret_cast<const uint32_t*>(&b);
        }
        if constexpr (V == 4) *reinterpret_cast<uint2*>(p) = make_uint2(w[0], w[1]);
        else *reinterpret_cast<uint32_t*>(p) = w[0];
    }
}

}  // namespace dlmk
