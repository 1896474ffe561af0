// One or four neighbouring entries of a row of either element type (or of the K-parts of a
// product), as floats: what the kernels that work on whole rows load and store at a time.
#pragma once
#include "common.cuh"

// N neighbouring values, converted.
template <int N>
struct Pack {
    float v[N];
};
template <int N>
__device__ __forceinline__ Pack<N> load_pack(const void* base, size_t i, int dtype) {
    Pack<N> r;
    if constexpr (N == 4) {
        if (dtype == MLS_BF16) {
            const uint2 raw = *reinterpret_cast<const uint2*>((const __nv_bfloat16*)base + i);
            const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
            const float2 a = __bfloat1622float2(h2[0]), b = __bfloat1622float2(h2[1]);
            r.v[0] = a.x; r.v[1] = a.y; r.v[2] = b.x; r.v[3] = b.y;
        } else {
            const float4 f = *reinterpret_cast<const float4*>((const float*)base + i);
            r.v[0] = f.x; r.v[1] = f.y; r.v[2] = f.z; r.v[3] = f.w;
        }
    } else {
        r.v[0] = load_as_float(base, i, dtype);
    }
    return r;
}
template <int N>
__device__ __forceinline__ Pack<N> load_parts(const void* base, size_t i, int dtype, int parts,
                                              size_t stride) {
    if (parts == 1) return load_pack<N>(base, i, dtype);
    Pack<N> s;
    if constexpr (N == 4) {
        const float4 f = sum_parts4<4>((const float*)base, i, parts, stride);
        s.v[0] = f.x; s.v[1] = f.y; s.v[2] = f.z; s.v[3] = f.w;
    } else {
        s.v[0] = ((const float*)base)[i];
        for (int k = 1; k < parts; ++k) s.v[0] += ((const float*)base)[i + k * stride];
    }
    return s;
}
template <int N>
__device__ __forceinline__ void store_pack(void* base, size_t i, int dtype, const Pack<N>& p) {
    if constexpr (N == 4) {
        const float4 f = make_float4(p.v[0], p.v[1], p.v[2], p.v[3]);
        if (dtype == MLS_BF16) *reinterpret_cast<uint2*>((__nv_bfloat16*)base + i) = pack_bf16x4(f);
        else *reinterpret_cast<float4*>((float*)base + i) = f;
    } else {
        store_from_float(base, i, dtype, p.v[0]);
    }
}
