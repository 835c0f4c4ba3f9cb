// A norm without statistics, fused with the residual sum in front of it:
//
//   h[t, :] <- h[t, :] + mult * (first[t, :] + second[t, :]);      out[t, :] = tanh(alpha h[t, :]) * w + b
//
// where the summands of the branch come as they are: a dense tensor, the unsummed float32 parts of a product whose contraction
// was cut, or rows of routed experts with a weight each (sum_k wts[t, k] * y[pair_row[t, k], :]).  Everything is element by
// element, so a row is cut over as many CTAs as the device has room for.  Sums, tanh and the stream are 32-bit; the parts of a
// product are added in split order, an expert's rows in the order of the choice.  With `rows`, output row r reads stream row
// rows[r] and the stream is left as it is.
#include <algorithm>

#include "common.cuh"

namespace {

struct DytTerm {
    const void* t;          // dense [T, d] in the activations' type, or null
    const float* parts;     // [n_splits][T, d], or null
    int n_splits;
    const void* y;          // rows of [*, d] in the activations' type, or null
    const int* pair_row;    // [T, top]
    const float* wts;       // [T, top]
    int top;
};

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

// VEC columns (4 or 1) of row `t` of a summand, added to acc.
template <typename TA, int VEC>
__device__ __forceinline__ void add_term(float (&acc)[VEC], const DytTerm& s, int64_t t, int c, int64_t d, int64_t n) {
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
        for (int k = 0; k < s.top; ++k) add((const TA*)s.y + (int64_t)s.pair_row[t * s.top + k] * d + c, s.wts[t * s.top + k]);
    } else if (s.t) {
        add((const TA*)s.t + t * d + c, 1.f);
    }
}

template <typename TA, typename TW, int VEC>
__global__ void __launch_bounds__(128) add_dyt_kernel(float* __restrict__ h, float mult, DytTerm first, DytTerm second, const float* __restrict__ alpha,
                                                      const TW* __restrict__ w, const TW* __restrict__ b, TA* __restrict__ out,
                                                      const int* __restrict__ rows, int64_t n_stream, int d, int write_h) {
    pdl_wait();
    pdl_launch_dependents();
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
    if (c >= d) return;
    const int64_t r = blockIdx.x, t = rows ? rows[r] : r;
    const int64_t n = n_stream * d;
    const float a = alpha[0];
    float x[VEC];
    if (VEC == 4) {
        const float4 v = *reinterpret_cast<const float4*>(h + t * d + c);
        x[0] = v.x, x[1 % VEC] = v.y, x[2 % VEC] = v.z, x[3 % VEC] = v.w;
    } else {
        x[0] = h[t * d + c];
    }
    const bool branch = first.t || first.parts || first.y || second.t || second.parts || second.y;
    if (branch) {
        float acc[VEC], acc2[VEC];
#pragma unroll
        for (int i = 0; i < VEC; ++i) acc[i] = acc2[i] = 0.f;
        add_term<TA, VEC>(acc, first, t, c, d, n);
        add_term<TA, VEC>(acc2, second, t, c, d, n);
#pragma unroll
        for (int i = 0; i < VEC; ++i) x[i] = fmaf(mult, acc[i] + acc2[i], x[i]);
        if (write_h) {
            if (VEC == 4) *reinterpret_cast<float4*>(h + t * d + c) = make_float4(x[0], x[1 % VEC], x[2 % VEC], x[3 % VEC]);
            else h[t * d + c] = x[0];
        }
    }
    float wv[VEC], bv[VEC];
    if (VEC == 4) {
        const float4 ww = Four<TW>::load(w + c), bb = Four<TW>::load(b + c);
        wv[0] = ww.x, wv[1 % VEC] = ww.y, wv[2 % VEC] = ww.z, wv[3 % VEC] = ww.w;
        bv[0] = bb.x, bv[1 % VEC] = bb.y, bv[2 % VEC] = bb.z, bv[3 % VEC] = bb.w;
    } else {
        wv[0] = to_float(w[c]), bv[0] = to_float(b[c]);
    }
#pragma unroll
    for (int i = 0; i < VEC; ++i) x[i] = fmaf(tanhf(a * x[i]), wv[i], bv[i]);
    if (VEC == 4) Four<TA>::store(out + r * d + c, make_float4(x[0], x[1 % VEC], x[2 % VEC], x[3 % VEC]));
    else out[r * d + c] = from_float<TA>(x[0]);
}

template <typename TA, typename TW>
cudaError_t launch_dyt(float* h, float mult, const DytTerm& a, const DytTerm& b2, const float* alpha, const void* w, const void* b, void* out,
                       const int* rows, int n_stream, int n_out, int d, int write_h, bool vec, cudaStream_t s) {
    const int per = vec ? 4 : 1, cols = (d + per - 1) / per;
    // few rows: small CTAs, so that a step of single tokens spreads over the device
    const int block = n_out <= 32 ? 64 : 128;
    const dim3 grid(n_out, (cols + block - 1) / block);
    if (vec)
        return imp_launch(add_dyt_kernel<TA, TW, 4>, grid, dim3(block), 0, s, h, mult, a, b2, alpha, (const TW*)w, (const TW*)b, (TA*)out, rows,
                          (int64_t)n_stream, d, write_h);
    return imp_launch(add_dyt_kernel<TA, TW, 1>, grid, dim3(block), 0, s, h, mult, a, b2, alpha, (const TW*)w, (const TW*)b, (TA*)out, rows,
                      (int64_t)n_stream, d, write_h);
}

}  // namespace

// The branch's two summands, each given as: t (dense), or parts with n_splits > 0, or y with pair_row, wts, top (all null: none).
// h float32 [n_stream, d]; w, b [d] of w_dtype; alpha float32 [1]; rows: null or [n_out] stream rows (then h is not written).
IMP_API int imp_add_dyt(float* h, float mult, const void* t1, const float* parts1, int n_splits1, const void* y1, const int* row1, const float* wts1,
                        int top1, const void* t2, const float* parts2, int n_splits2, const void* y2, const int* row2, const float* wts2, int top2,
                        const float* alpha, const void* w, const void* b, void* out, const int* rows, int n_stream, int n_out, int d,
                        int act_dtype, int w_dtype, void* stream) {
    if (n_out == 0) return 0;
    IMP_CHECK_ARG(h && alpha && w && b && out && d > 0 && n_stream > 0, "imp_add_dyt: bad argument");
    IMP_CHECK_ARG(rows || n_out == n_stream, "imp_add_dyt: without a row list every stream row is an output row");
    IMP_CHECK_ARG((!y1 || (row1 && wts1 && top1 > 0)) && (!y2 || (row2 && wts2 && top2 > 0)), "imp_add_dyt: routed rows need their places and weights");
    const DytTerm a{t1, parts1, n_splits1, y1, row1, wts1, top1}, c{t2, parts2, n_splits2, y2, row2, wts2, top2};
    bool vec = d % 4 == 0;
    for (const void* p : {(const void*)h, t1, (const void*)parts1, y1, t2, (const void*)parts2, y2, w, b, (const void*)out}) vec = vec && (uintptr_t)p % 16 == 0;
    cudaStream_t s = (cudaStream_t)stream;
    const int write_h = rows ? 0 : 1;
    cudaError_t e;
    if (act_dtype == IMP_F32)
        e = w_dtype == IMP_F32 ? launch_dyt<float, float>(h, mult, a, c, alpha, w, b, out, rows, n_stream, n_out, d, write_h, vec, s)
                               : launch_dyt<float, __nv_bfloat16>(h, mult, a, c, alpha, w, b, out, rows, n_stream, n_out, d, write_h, vec, s);
    else
        e = w_dtype == IMP_F32 ? launch_dyt<__nv_bfloat16, float>(h, mult, a, c, alpha, w, b, out, rows, n_stream, n_out, d, write_h, vec, s)
                               : launch_dyt<__nv_bfloat16, __nv_bfloat16>(h, mult, a, c, alpha, w, b, out, rows, n_stream, n_out, d, write_h, vec, s);
    if (e != cudaSuccess) {
        imp_set_error("imp_add_dyt: %s", cudaGetErrorString(e));
        return (int)e;
    }
    return 0;
}
