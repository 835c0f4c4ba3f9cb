// Reading a summand of a branch (ImpBranchTerm) four columns at a time or one by one, in 32-bit.
#pragma once

#include "branch_terms.h"
#include "common.cuh"

template <typename TA> struct Four {};
template <> struct Four<float> {
    static __device__ __forceinline__ float4 load(const float* p) { return *reinterpret_cast<const float4*>(p); }
    static __device__ __forceinline__ void store(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
};
template <> struct Four<__nv_bfloat16> {
    static __device__ __forceinline__ float4 load(const __nv_bfloat16* p) {
        const uint2 u = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
        return make_float4(a.x, a.y, b.x, b.y);
    }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, float4 v) {
        __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
        uint2 u;
        u.x = *reinterpret_cast<uint32_t*>(&a), u.y = *reinterpret_cast<uint32_t*>(&b);
        *reinterpret_cast<uint2*>(p) = u;
    }
};

// VEC columns (4 or 1) from column c on of row t of a summand, added to acc; `self`: the stream's values there; n = T * d.
template <typename TA, int VEC>
__device__ __forceinline__ void add_term(float (&acc)[VEC], const ImpBranchTerm& s, const float (&self)[VEC], int64_t t, int c, int64_t d, int64_t n) {
    auto add = [&](const TA* p, float f) {
        if (VEC == 4) {
            const float4 v = Four<TA>::load(p);
            acc[0] = fmaf(f, v.x, acc[0]), acc[1 % VEC] = fmaf(f, v.y, acc[1 % VEC]), acc[2 % VEC] = fmaf(f, v.z, acc[2 % VEC]), acc[3 % VEC] = fmaf(f, v.w, acc[3 % VEC]);
        } else {
            acc[0] = fmaf(f, to_float(*p), acc[0]);
        }
    };
    if (s.parts) {
        const float* p = s.parts + t * d + c;
#pragma unroll 4
        for (int i = 0; i < s.n_splits; ++i, p += n) {
            if (VEC == 4) {
                const float4 v = *reinterpret_cast<const float4*>(p);
                acc[0] += v.x, acc[1 % VEC] += v.y, acc[2 % VEC] += v.z, acc[3 % VEC] += v.w;
            } else {
                acc[0] += *p;
            }
        }
    } else if (s.y) {
#pragma unroll 4
        for (int k = 0; k < s.top; ++k) {
            const int row = s.pair_row[t * s.top + k];
            const float f = s.wts[t * s.top + k];
            if (row >= 0) {
                add((const TA*)s.y + (int64_t)row * d + c, f);
            } else if (s.input) {
                add((const TA*)s.input + t * d + c, f);
            } else {
#pragma unroll
                for (int i = 0; i < VEC; ++i) acc[i] = fmaf(f, self[i], acc[i]);
            }
        }
    } else if (s.t) {
        add((const TA*)s.t + t * d + c, 1.f);
    }
}

// Every pointer of a summand starts on 16 bytes (what four columns at a time need, with d a multiple of 4).
inline bool term_aligned(const ImpBranchTerm& s) {
    for (const void* p : {s.t, (const void*)s.parts, s.y, s.input})
        if ((uintptr_t)p % 16) return false;
    return true;
}
inline bool term_valid(const ImpBranchTerm& s) { return !s.y || (s.pair_row && s.wts && s.top > 0); }
