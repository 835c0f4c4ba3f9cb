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

// The same for a thread that holds NV pieces of four columns, piece i from column first + i * step on while that is below d: what a
// thread needs of all its pieces is asked for together, parts of a product several at a time, and added in the same order.
// PARTS: the summand may be a product's parts.
template <typename TA, int NV, bool PARTS>
__device__ __forceinline__ void add_term_pieces(float (&acc)[NV][4], const ImpBranchTerm& s, const float (&self)[NV][4], int64_t t, int first, int step, int d,
                                                int64_t n) {
    auto fma4 = [](float (&a)[4], float f, const float4& v) {
        a[0] = fmaf(f, v.x, a[0]), a[1] = fmaf(f, v.y, a[1]), a[2] = fmaf(f, v.z, a[2]), a[3] = fmaf(f, v.w, a[3]);
    };
    if (PARTS && s.parts) {
        constexpr int NB = NV == 1 ? 12 : NV == 2 ? 6 : 2;
        const float* p = s.parts + t * d;
        for (int s0 = 0; s0 < s.n_splits; s0 += NB) {
            float4 v[NB][NV];
#pragma unroll
            for (int j = 0; j < NB; ++j)
#pragma unroll
                for (int i = 0; i < NV; ++i)
                    if (s0 + j < s.n_splits && first + i * step < d) v[j][i] = *reinterpret_cast<const float4*>(p + (s0 + j) * n + first + i * step);
#pragma unroll
            for (int j = 0; j < NB; ++j)
#pragma unroll
                for (int i = 0; i < NV; ++i)
                    if (s0 + j < s.n_splits && first + i * step < d) acc[i][0] += v[j][i].x, acc[i][1] += v[j][i].y, acc[i][2] += v[j][i].z, acc[i][3] += v[j][i].w;
        }
    } else if (s.y) {
        for (int k = 0; k < s.top; ++k) {
            const int row = s.pair_row[t * s.top + k];
            const float f = s.wts[t * s.top + k];
            const TA* src = row >= 0 ? (const TA*)s.y + (int64_t)row * d : s.input ? (const TA*)s.input + t * d : nullptr;
            if (src) {
                float4 v[NV];
#pragma unroll
                for (int i = 0; i < NV; ++i)
                    if (first + i * step < d) v[i] = Four<TA>::load(src + first + i * step);
#pragma unroll
                for (int i = 0; i < NV; ++i)
                    if (first + i * step < d) fma4(acc[i], f, v[i]);
            } else {
#pragma unroll
                for (int i = 0; i < NV; ++i)
#pragma unroll
                    for (int e = 0; e < 4; ++e) acc[i][e] = fmaf(f, self[i][e], acc[i][e]);
            }
        }
    } else if (s.t) {
        const TA* src = (const TA*)s.t + t * d;
#pragma unroll
        for (int i = 0; i < NV; ++i)
            if (first + i * step < d) fma4(acc[i], 1.f, Four<TA>::load(src + first + i * step));
    }
}

// Every pointer of a summand starts on 16 bytes (what four columns at a time need, with d a multiple of 4).
inline bool term_aligned(const ImpBranchTerm& s) {
    for (const void* p : {s.t, (const void*)s.parts, s.y, s.input})
        if ((uintptr_t)p % 16) return false;
    return true;
}
inline bool term_valid(const ImpBranchTerm& s) { return !s.y || (s.pair_row && s.wts && s.top > 0); }
