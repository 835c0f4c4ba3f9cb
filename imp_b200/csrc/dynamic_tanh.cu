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

#include "branch_terms.cuh"
#include "common.cuh"

namespace {

template <typename TA, typename TW, int VEC>
__global__ void __launch_bounds__(128) add_dyt_kernel(float* __restrict__ h, float mult, ImpBranchTerm first, ImpBranchTerm second, const float* __restrict__ alpha,
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
        add_term<TA, VEC>(acc, first, x, t, c, d, n);
        add_term<TA, VEC>(acc2, second, x, t, c, d, n);
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
cudaError_t launch_dyt(float* h, float mult, const ImpBranchTerm& a, const ImpBranchTerm& b2, const float* alpha, const void* w, const void* b, void* out,
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

// The branch's two summands (branch_terms.h; all null: none).  h float32 [n_stream, d]; w, b [d] of w_dtype; alpha float32 [1];
// rows: null or [n_out] stream rows (then h is not written).
IMP_API int imp_add_dyt(float* h, float mult, const ImpBranchTerm* first, const ImpBranchTerm* second, const float* alpha, const void* w,
                        const void* b, void* out, const int* rows, int n_stream, int n_out, int d, int act_dtype, int w_dtype, void* stream) {
    if (n_out == 0) return 0;
    IMP_CHECK_ARG(h && first && second && alpha && w && b && out && d > 0 && n_stream > 0, "imp_add_dyt: bad argument");
    IMP_CHECK_ARG(rows || n_out == n_stream, "imp_add_dyt: without a row list every stream row is an output row");
    const ImpBranchTerm a = *first, c = *second;
    IMP_CHECK_ARG(term_valid(a) && term_valid(c), "imp_add_dyt: routed rows need their places and weights");
    bool vec = d % 4 == 0 && term_aligned(a) && term_aligned(c);
    for (const void* p : {(const void*)h, w, b, (const void*)out}) vec = vec && (uintptr_t)p % 16 == 0;
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
