// Rows of a matrix product as the kernel after it reads them: an array of either element type, or the 32-bit
// partial sums [splits][rows][columns] of a product whose K range was split, added up in split order on the way.
#pragma once

#include "common.cuh"

namespace chibi {

// V neighbouring values (V = 1, 4, or 8 for 16-bit types) in one access; aligned to V values.
template <typename T, int V>
__device__ __forceinline__ void load_values(float (&dst)[V], const T* src)
{
    if constexpr (V == 1) {
        dst[0] = to_f32(src[0]);
    } else if constexpr (sizeof(T) == 4) {
#pragma unroll
        for (int i = 0; i < V; i += 4) {
            const float4 v = *reinterpret_cast<const float4*>(src + i);
            dst[i] = v.x, dst[i + 1] = v.y, dst[i + 2] = v.z, dst[i + 3] = v.w;
        }
    } else {
        uint32_t w[V / 2];
        if constexpr (V == 8) {
            const uint4 v = *reinterpret_cast<const uint4*>(src);
            w[0] = v.x, w[1] = v.y, w[2] = v.z, w[3] = v.w;
        } else {
            const uint2 v = *reinterpret_cast<const uint2*>(src);
            w[0] = v.x, w[1] = v.y;
        }
#pragma unroll
        for (int i = 0; i < V / 2; ++i) {
            const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w[i]));
            dst[2 * i] = f.x, dst[2 * i + 1] = f.y;
        }
    }
}

template <typename T, int V>
__device__ __forceinline__ void store_values(T* dst, const float (&src)[V])
{
    if constexpr (V == 1) {
        dst[0] = from_f32<T>(src[0]);
    } else if constexpr (sizeof(T) == 4) {
#pragma unroll
        for (int i = 0; i < V; i += 4)
            *reinterpret_cast<float4*>(dst + i) = make_float4(src[i], src[i + 1], src[i + 2], src[i + 3]);
    } else {
        uint32_t w[V / 2];
#pragma unroll
        for (int i = 0; i < V / 2; ++i) {
            const __nv_bfloat162 h = __floats2bfloat162_rn(src[2 * i], src[2 * i + 1]);
            w[i] = *reinterpret_cast<const uint32_t*>(&h);
        }
        if constexpr (V == 8)
            *reinterpret_cast<uint4*>(dst) = make_uint4(w[0], w[1], w[2], w[3]);
        else
            *reinterpret_cast<uint2*>(dst) = make_uint2(w[0], w[1]);
    }
}

template <typename T>
struct ProductRows {
    const T* base;
    long long stride;          // from row to row
    int splits;                // 1: `base` is the product itself
    long long split_stride;

    // columns c .. c + V - 1 of row t
    template <int V>
    __device__ __forceinline__ void load(float (&dst)[V], long long t, int c) const
    {
        const T* p = base + t * stride + c;
        load_values<T, V>(dst, p);
        for (int s = 1; s < splits; s += 4) {
            float more[4][V];
#pragma unroll
            for (int k = 0; k < 4; ++k)
                if (s + k < splits)
                    load_values<T, V>(more[k], p + (s + k) * split_stride);
#pragma unroll
            for (int k = 0; k < 4; ++k)
                if (s + k < splits) {
#pragma unroll
                    for (int i = 0; i < V; ++i)
                        dst[i] += more[k][i];
                }
        }
    }
    __device__ __forceinline__ float at(long long t, int c) const
    {
        float v[1];
        load<1>(v, t, c);
        return v[0];
    }
};

// Whether rows of `type` that start at `base` can be read four values at a time.
inline bool rows_in_fours(const void* base, int type, long long stride, long long split_stride)
{
    return stride % 4 == 0 && split_stride % 4 == 0
           && reinterpret_cast<uintptr_t>(base) % (type == CHIBI_F32 ? 16 : 8) == 0;
}

} // namespace chibi
