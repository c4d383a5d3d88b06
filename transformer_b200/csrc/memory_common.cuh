// What the kernels of the linear memories (decay_memory.cu, gated_linear.cu, split_delta.cu) share.
#pragma once
#include "common.cuh"

// rows of a memory that a scan's lanes cover for heads of `dim` key channels
__host__ __device__ inline int dm_rows(int dim) { return dim <= 16 ? 16 : dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : 256; }

template <typename T, int V>
__device__ __forceinline__ void dm_load(const T* p, float (&f)[V]) {
    if constexpr (V == 1) {
        f[0] = ldf(p);
    } else if constexpr (sizeof(T) == 2) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
    } else {
        const float4 a = *reinterpret_cast<const float4*>(p);
        f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
    }
}
template <int V>
__device__ __forceinline__ void dm_store(float* p, const float (&f)[V]) {
    if constexpr (V == 1) *p = f[0];
    else *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
}

// This lane's share of W2 row . ta: `parts` adjacent lanes take a row's pieces of eight (or entries) in turn.
template <typename T>
__device__ __forceinline__ float decay_dot(const T* __restrict__ w2row, const float* ta, int rank, int part, int parts) {
    float acc = 0.f;
    if ((rank & 7) == 0) {
#pragma unroll 4
        for (int q = part * 8; q < rank; q += parts * 8) {
            float w[8];
            load8(w2row + q, w);
            const float4 t0 = *reinterpret_cast<const float4*>(ta + q);
            const float4 t1 = *reinterpret_cast<const float4*>(ta + q + 4);
            acc += w[0] * t0.x + w[1] * t0.y + w[2] * t0.z + w[3] * t0.w + w[4] * t1.x + w[5] * t1.y + w[6] * t1.z + w[7] * t1.w;
        }
        return acc;
    }
    for (int q = part; q < rank; q += parts) acc += ldf(w2row + q) * ta[q];
    return acc;
}

// two floats in one register pair, and the hardware's packed multiply-add on them
union F2 {
    float2 f;
    unsigned long long u;
};
__device__ __forceinline__ F2 fma2(F2 a, F2 b, F2 c) {
    F2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d.u) : "l"(a.u), "l"(b.u), "l"(c.u));
    return d;
}
__device__ __forceinline__ F2 mul2(F2 a, F2 b) {
    F2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d.u) : "l"(a.u), "l"(b.u));
    return d;
}

