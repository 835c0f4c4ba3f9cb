// RMS norms of what a sublayer gives, joined with the residual sum, and of a token's embedding:
//
//   add_rms_branch       b = first + second + bias (32-bit);  h <- h + b / sqrt(mean(b^2) + eps) * w;  out = h
//   embedding_rmsnorm    e = table[id] * scale;               h  = e / sqrt(mean(e^2) + eps) * w;      out = h
//
// h is the 32-bit residual stream, `out` its copy in the activations' type, which the next sublayer reads.  The summands come
// as they are (branch_terms.h): dense tensors, unsummed parts of a product, rows of routed experts with their weights, identity
// experts among them, so no kernel stands between the products and this one.  Sums, statistics and the stream are 32-bit and
// nothing is rounded on the way.
//
// add_rms_branch has three forms.  Rows in registers, a CTA a row.  For few rows, a cluster of up to 8 CTAs shares a row, so
// that a product's parts are fetched by enough threads at once: each CTA adds up its squares and stores the sum into every
// CTA of the cluster (distributed shared memory), and after one cluster barrier all of them add the same numbers in rank order.
// And one column at a time, reading the branch twice, for widths that are no multiple of 4 or beyond the registers.  In the
// float32 path the form depends on the width alone, so a row's result does not depend on what else is in the batch.
#include "branch_terms.cuh"
#include "common.cuh"

namespace {

constexpr int BN_THREADS = 128, BN_MAX_C = 8, BN_ROW_THREADS = 256;


// NV float4 a thread; CLUSTER: gridDim.x / C rows, a cluster of C CTAs each; else a CTA a row.  FORM: what the branch is, so that the usual
// cases of long portions need few registers: any, one dense tensor (asked for together with the stream), or no unsummed parts.
enum : int { BN_ANY = 0, BN_DENSE = 1, BN_NO_PARTS = 2 };
template <typename TA, typename TW, int NV, bool CLUSTER, int FORM>
__global__ void __launch_bounds__(CLUSTER ? BN_THREADS : BN_ROW_THREADS)
    add_rms_branch_kernel(float* __restrict__ h, ImpBranchTerm first, ImpBranchTerm second, const float* __restrict__ bias, const TW* __restrict__ w,
                          TA* __restrict__ out, int64_t n_rows, int d, float eps, int C) {
    constexpr bool DENSE = FORM == BN_DENSE;
    constexpr int NT = CLUSTER ? BN_THREADS : BN_ROW_THREADS;
    __shared__ float scratch[33];
    __shared__ float slots[BN_MAX_C];
    // first half of "every CTA of the cluster is running"; the wait stands before the first remote store
    if (CLUSTER) asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");
    pdl_wait();
    pdl_launch_dependents();
    const int rank = CLUSTER ? blockIdx.x % C : 0;
    const int64_t t = CLUSTER ? blockIdx.x / C : blockIdx.x;
    const int nv = d >> 2, stride = (CLUSTER ? C : 1) * NT;
    float* hrow = h + t * d;
    float x[NV][4], b[NV][4];
    float4 wv[NV];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = rank * NT + threadIdx.x + i * stride;
        if (c < nv) {
            const float4 v = *reinterpret_cast<const float4*>(hrow + 4 * c);
            x[i][0] = v.x, x[i][1] = v.y, x[i][2] = v.z, x[i][3] = v.w;
            if (DENSE) {
                const float4 y = Four<TA>::load((const TA*)first.t + t * d + 4 * c);
                b[i][0] = y.x, b[i][1] = y.y, b[i][2] = y.z, b[i][3] = y.w;
            }
            wv[i] = Four<TW>::load(w + 4 * c);
            if (DENSE && !bias) continue;
            const float4 b0 = bias ? *reinterpret_cast<const float4*>(bias + 4 * c) : make_float4(0.f, 0.f, 0.f, 0.f);
            if (DENSE) b[i][0] += b0.x, b[i][1] += b0.y, b[i][2] += b0.z, b[i][3] += b0.w;
            else b[i][0] = b0.x, b[i][1] = b0.y, b[i][2] = b0.z, b[i][3] = b0.w;
        }
    }
    if (!DENSE) {
        const int c0 = 4 * (rank * NT + (int)threadIdx.x);
        add_term_pieces<TA, NV, FORM == BN_ANY>(b, first, x, t, c0, 4 * stride, d, n_rows * d);
        add_term_pieces<TA, NV, FORM == BN_ANY>(b, second, x, t, c0, 4 * stride, d, n_rows * d);
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = rank * NT + threadIdx.x + i * stride;
        if (c < nv) {
#pragma unroll
            for (int e = 0; e < 4; ++e) ss = fmaf(b[i][e], b[i][e], ss);
        }
    }
    ss = block_sum(ss, scratch);
    if (CLUSTER) {
        asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
        if (threadIdx.x < C) {
            const uint32_t local = (uint32_t)__cvta_generic_to_shared(&slots[rank]);
            uint32_t remote;
            asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local), "r"((uint32_t)threadIdx.x));
            asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(remote), "f"(ss) : "memory");
        }
        asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
        asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
        ss = 0.f;
        for (int k = 0; k < C; ++k) ss += slots[k];
    }
    const float r = rsqrtf(ss / (float)d + eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = rank * NT + threadIdx.x + i * stride;
        if (c < nv) {
            const float4 v = make_float4(fmaf(b[i][0] * r, wv[i].x, x[i][0]), fmaf(b[i][1] * r, wv[i].y, x[i][1]), fmaf(b[i][2] * r, wv[i].z, x[i][2]),
                                         fmaf(b[i][3] * r, wv[i].w, x[i][3]));
            *reinterpret_cast<float4*>(hrow + 4 * c) = v;
            Four<TA>::store(out + t * d + 4 * c, v);
        }
    }
}

template <typename TA, typename TW>
__global__ void __launch_bounds__(BN_ROW_THREADS) add_rms_branch_scalar_kernel(float* __restrict__ h, ImpBranchTerm first, ImpBranchTerm second,
                                                                              const float* __restrict__ bias, const TW* __restrict__ w,
                                                                              TA* __restrict__ out, int64_t n_rows, int d, float eps) {
    pdl_wait();
    pdl_launch_dependents();
    __shared__ float scratch[33];
    const int64_t t = blockIdx.x;
    float* hrow = h + t * d;
    auto value = [&](int c, float x) {
        float b[1] = {bias ? bias[c] : 0.f};
        const float self[1] = {x};
        add_term<TA, 1>(b, first, self, t, c, d, n_rows * d);
        add_term<TA, 1>(b, second, self, t, c, d, n_rows * d);
        return b[0];
    };
    float ss = 0.f;
    for (int c = threadIdx.x; c < d; c += BN_ROW_THREADS) {
        const float b = value(c, hrow[c]);
        ss = fmaf(b, b, ss);
    }
    const float r = rsqrtf(block_sum(ss, scratch) / (float)d + eps);
    for (int c = threadIdx.x; c < d; c += BN_ROW_THREADS) {   // a thread rewrites what it alone has read
        const float x = hrow[c];
        const float v = fmaf(value(c, x) * r, to_float(w[c]), x);
        hrow[c] = v;
        out[t * d + c] = from_float<TA>(v);
    }
}

template <typename TA, typename TW>
cudaError_t launch_branch(float* h, const ImpBranchTerm& a, const ImpBranchTerm& b, const float* bias, const void* w, void* out, int n, int d, float eps,
                          bool vec, cudaStream_t s) {
    const int nv = d / 4;
    if (!vec || nv > BN_ROW_THREADS * 8)
        return imp_launch(add_rms_branch_scalar_kernel<TA, TW>, dim3(n), dim3(BN_ROW_THREADS), 0, s, h, a, b, bias, (const TW*)w, (TA*)out, (int64_t)n, d, eps);
    const int want = (nv + BN_THREADS - 1) / BN_THREADS;
    if (sizeof(TA) == 2 && n <= 64 && want > 1 && want <= 2 * BN_MAX_C) {
        const int per = want > BN_MAX_C ? 2 : 1, C = (want + per - 1) / per;
        cudaLaunchConfig_t cfg = {};
        cfg.gridDim = dim3((unsigned)(C * n));
        cfg.blockDim = dim3(BN_THREADS);
        cfg.stream = s;
        cudaLaunchAttribute attr[2];
        attr[0].id = cudaLaunchAttributeClusterDimension;
        attr[0].val.clusterDim.x = (unsigned)C;
        attr[0].val.clusterDim.y = 1;
        attr[0].val.clusterDim.z = 1;
        attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[1].val.programmaticStreamSerializationAllowed = 1;
        cfg.attrs = attr;
        cfg.numAttrs = imp_pdl_enabled() ? 2 : 1;
        if (per == 1)
            return cudaLaunchKernelEx(&cfg, add_rms_branch_kernel<TA, TW, 1, true, BN_ANY>, h, a, b, bias, (const TW*)w, (TA*)out, (int64_t)n, d, eps, C);
        return cudaLaunchKernelEx(&cfg, add_rms_branch_kernel<TA, TW, 2, true, BN_ANY>, h, a, b, bias, (const TW*)w, (TA*)out, (int64_t)n, d, eps, C);
    }
    const int per = (nv + BN_ROW_THREADS - 1) / BN_ROW_THREADS;
    const int form = a.parts || b.parts ? BN_ANY : a.t && !b.t && !b.y ? BN_DENSE : BN_NO_PARTS;
#define BN_ROW(NV) (form == BN_DENSE ? BN_ROW_FORM(NV, BN_DENSE) : form == BN_NO_PARTS ? BN_ROW_FORM(NV, BN_NO_PARTS) : BN_ROW_FORM(NV, BN_ANY))
#define BN_ROW_FORM(NV, FORM) \
    imp_launch(add_rms_branch_kernel<TA, TW, NV, false, FORM>, dim3(n), dim3(BN_ROW_THREADS), 0, s, h, a, b, bias, (const TW*)w, (TA*)out, (int64_t)n, d, eps, 1)
    return per <= 1 ? BN_ROW(1) : per <= 2 ? BN_ROW(2) : per <= 4 ? BN_ROW(4) : BN_ROW(8);
#undef BN_ROW
#undef BN_ROW_FORM
}

// A CTA per token; four columns a thread where the rows allow it (vec), else one.
template <typename TA, typename TE, typename TW>
__global__ void __launch_bounds__(BN_ROW_THREADS) embedding_rmsnorm_kernel(float* __restrict__ h, TA* __restrict__ out, const TE* __restrict__ table,
                                                                          const int* __restrict__ ids, const TW* __restrict__ w, int d, int vocab,
                                                                          float scale, float eps, int vec, int* status) {
    pdl_wait();
    pdl_launch_dependents();
    __shared__ float scratch[33];
    const int64_t t = blockIdx.x;
    const int id = ids[t];
    const bool bad = id < 0 || id >= vocab;
    if (bad && threadIdx.x == 0) imp_report(status, IMP_BAD_TOKEN_ID);
    const TE* row = table + (int64_t)(bad ? 0 : id) * d;
    const float f = bad ? 0.f : scale;
    float ss = 0.f;
    if (vec) {
        for (int c = threadIdx.x * 4; c < d; c += BN_ROW_THREADS * 4) {
            const float4 v = Four<TE>::load(row + c);
            const float4 e = make_float4(v.x * f, v.y * f, v.z * f, v.w * f);
            ss += (e.x * e.x + e.y * e.y) + (e.z * e.z + e.w * e.w);
        }
    } else {
        for (int c = threadIdx.x; c < d; c += BN_ROW_THREADS) {
            const float e = to_float(row[c]) * f;
            ss = fmaf(e, e, ss);
        }
    }
    const float r = rsqrtf(block_sum(ss, scratch) / (float)d + eps) * f;
    if (vec) {
        for (int c = threadIdx.x * 4; c < d; c += BN_ROW_THREADS * 4) {
            const float4 v = Four<TE>::load(row + c), ww = Four<TW>::load(w + c);
            const float4 o = make_float4(v.x * r * ww.x, v.y * r * ww.y, v.z * r * ww.z, v.w * r * ww.w);
            *reinterpret_cast<float4*>(h + t * d + c) = o;
            Four<TA>::store(out + t * d + c, o);
        }
    } else {
        for (int c = threadIdx.x; c < d; c += BN_ROW_THREADS) {
            const float o = to_float(row[c]) * r * to_float(w[c]);
            h[t * d + c] = o;
            out[t * d + c] = from_float<TA>(o);
        }
    }
}

int failed(const char* what, cudaError_t e) {
    imp_set_error("%s: %s", what, cudaGetErrorString(e));
    return (int)e;
}

}  // namespace

// h float32 [n, d] (updated); first, second: the branch's summands over its n rows; bias float32 [d] or null; w [d] of w_dtype;
// out [n, d] of act_dtype.
IMP_API int imp_add_rms_branch(float* h, const ImpBranchTerm* first, const ImpBranchTerm* second, const float* bias, const void* w, void* out, int n,
                               int d, float eps, int act_dtype, int w_dtype, void* stream) {
    if (n == 0) return 0;
    IMP_CHECK_ARG(h && first && second && w && out && n > 0 && d > 0, "imp_add_rms_branch: bad argument");
    const ImpBranchTerm a = *first, b = *second;
    IMP_CHECK_ARG(term_valid(a) && term_valid(b), "imp_add_rms_branch: routed rows need their places and weights");
    bool vec = d % 4 == 0 && term_aligned(a) && term_aligned(b);
    for (const void* p : {(const void*)h, (const void*)bias, w, (const void*)out}) vec = vec && (uintptr_t)p % 16 == 0;
    cudaStream_t s = (cudaStream_t)stream;
    cudaError_t e;
    if (act_dtype == IMP_F32)
        e = w_dtype == IMP_F32 ? launch_branch<float, float>(h, a, b, bias, w, out, n, d, eps, vec, s)
                               : launch_branch<float, __nv_bfloat16>(h, a, b, bias, w, out, n, d, eps, vec, s);
    else
        e = w_dtype == IMP_F32 ? launch_branch<__nv_bfloat16, float>(h, a, b, bias, w, out, n, d, eps, vec, s)
                               : launch_branch<__nv_bfloat16, __nv_bfloat16>(h, a, b, bias, w, out, n, d, eps, vec, s);
    return e == cudaSuccess ? 0 : failed("imp_add_rms_branch", e);
}

// h float32 [n, d] and out [n, d] (act_dtype) from rows ids[t] of the table [vocab, d]; w [d].
IMP_API int imp_embedding_rmsnorm(float* h, void* out, const void* table, const int* ids, const void* w, int n, int d, int vocab, float scale,
                                  float eps, int act_dtype, int table_dtype, int w_dtype, int* status, void* stream) {
    if (n == 0) return 0;
    IMP_CHECK_ARG(h && out && table && ids && w && n > 0 && d > 0 && vocab > 0, "imp_embedding_rmsnorm: bad argument");
    int vec = d % 4 == 0;
    for (const void* p : {(const void*)h, (const void*)out, table, w}) vec = vec && (uintptr_t)p % 16 == 0;
    cudaStream_t s = (cudaStream_t)stream;
    cudaError_t e;
#define EN(TA, TE, TW)                                                                                                                          \
    imp_launch(embedding_rmsnorm_kernel<TA, TE, TW>, dim3(n), dim3(BN_ROW_THREADS), 0, s, h, (TA*)out, (const TE*)table, ids, (const TW*)w, d, vocab, \
               scale, eps, vec, status)
    using bf = __nv_bfloat16;
    if (act_dtype == IMP_F32)
        e = table_dtype == IMP_F32 ? (w_dtype == IMP_F32 ? EN(float, float, float) : EN(float, float, bf))
                                   : (w_dtype == IMP_F32 ? EN(float, bf, float) : EN(float, bf, bf));
    else
        e = table_dtype == IMP_F32 ? (w_dtype == IMP_F32 ? EN(bf, float, float) : EN(bf, float, bf))
                                   : (w_dtype == IMP_F32 ? EN(bf, bf, float) : EN(bf, bf, bf));
#undef EN
    return e == cudaSuccess ? 0 : failed("imp_embedding_rmsnorm", e);
}
