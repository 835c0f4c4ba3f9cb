// Routing of a mixture of experts, and the sum of the chosen experts' outputs.
//
//   z[t, e]   = x[t] . Wr[e] + b[e]                       32-bit
//   chosen    = the `top` experts with the largest z (the lower index wins a tie)
//   weight    = softmax over the chosen logits only; or, with sigmoid scores s = sigmoid(z): weight = s * weight_scale
//               or, with softmax scores over all experts: weight = that softmax * weight_scale, not renormalised
//               or, with softmax scores and a bias on the choice: the `top` largest softmax + c[e] choose, the weight is the
//               softmax without c, optionally divided by the chosen ones' sum (+ 1e-20)
//   groups    = optionally the experts form n_groups equal groups of neighbours; a group's score is the sum of its two
//               largest scores, or its largest one, and only the experts of the `keep` best groups can be chosen
//   gate[t]   = sigmoid(x[t] . Wg)                         one number per token, for a shared expert (optional)
//   out[t]    = sum_k weight[t, k] * y[place(t, k)] + gate[t] * shared[t]
// Router outputs beyond the experts that have matrices are identity experts: they are chosen and weighed like the others, take no
// part in the list (place -1), and give the input itself, y = x[t].
//
// Where the router's weights are 16-bit the logits come from the tensor-core product (16-bit operands, 32-bit sums and results: what
// the 32-bit product of the same numbers gives up to the order of its sum) and moe_choose makes the choice; otherwise moe_route does both.
//
// The expert products run over a list of (token, choice) pairs sorted by expert (see grouped_gemm.cu); moe_sort makes
// that list on the device: seg [E + 1], the token of every list row, and the row of every pair.  Nothing comes back
// to the host, so the launches of a step depend on its sizes alone.
#include "common.cuh"

namespace {

template <typename T> struct Vec4 {};
template <> struct Vec4<float> {
    static __device__ __forceinline__ float4 load(const float* p) { return *reinterpret_cast<const float4*>(p); }
    static __device__ __forceinline__ void store(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
};
template <> struct Vec4<__nv_bfloat16> {
    static __device__ __forceinline__ float4 load(const __nv_bfloat16* p) {
        const uint2 u = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
        return make_float4(a.x, a.y, b.x, b.y);
    }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, float4 v) {
        __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
        uint2 u;
        u.x = *reinterpret_cast<uint32_t*>(&a);
        u.y = *reinterpret_cast<uint32_t*>(&b);
        *reinterpret_cast<uint2*>(p) = u;
    }
};

constexpr int ROUTE_BLOCK = 256, ROUTE_MAX_E = 1024, ROUTE_MAX_TOP = 32;

// The choice of one token, made by one warp: `top` rounds of arg-max over what is left (the lower index wins a tie), and the
// weights.  zt [E] in shared memory: the logits, or with score_mode 1 the sigmoid scores; gt [n_groups] and cs [E] (with
// choice_bias): room for the groups' and the biased scores.  idx, wts [top].
struct RouteRule {
    int E, top, score_mode, n_groups, keep, group_top;
    float weight_scale;
    const float* choice_bias;
    int renormalise;
};
__device__ __forceinline__ void choose_experts(const RouteRule& p, float* zt, float* gt, float* cs, int lane, int* __restrict__ idx, float* __restrict__ wts) {
    const int E = p.E, top = p.top;
    const float* zl = zt;            // the logits, where the choice scores are others
    float chosen[ROUTE_MAX_TOP];
    // softmax scores: the choice runs on the logits (same order); the weights need the largest and the sum over all experts
    float z_max = 0.f, z_sum = 1.f;
    if (p.score_mode == 2) {
        float m = -INFINITY;
        for (int e = lane; e < E; e += 32) m = fmaxf(m, zt[e]);
        z_max = warp_max(m);
        float sum = 0.f;
        for (int e = lane; e < E; e += 32) sum += expf(zt[e] - z_max);
        z_sum = warp_sum(sum);
        if (p.choice_bias) {
            zt = cs;
            for (int e = lane; e < E; e += 32) zt[e] = expf(zl[e] - z_max) / z_sum + p.choice_bias[e];
        }
        __syncwarp();
    }
    if (p.n_groups > 0) {
        // a group's score: the sum of its two largest scores (of its one score where a group is one expert),
        // or with group_top 1 its largest one; then `keep`
        // rounds of arg-max over the groups, the lower index winning a tie; the experts of the other groups leave
        const int per = E / p.n_groups;
        for (int g = lane; g < p.n_groups; g += 32) {
            float a = -INFINITY, b = -INFINITY;
            for (int e = g * per; e < (g + 1) * per; ++e) {
                const float v = zt[e];
                if (v > a) b = a, a = v;
                else if (v > b) b = v;
            }
            gt[g] = per > 1 && p.group_top == 2 ? a + b : a;
        }
        __syncwarp();
        for (int k = 0; k < p.keep; ++k) {
            float best = -INFINITY;
            int at = 0x7fffffff;
            for (int g = lane; g < p.n_groups; g += 32) {
                const float v = gt[g];
                if (v > best) best = v, at = g;
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) {
                const float ov = __shfl_xor_sync(0xffffffffu, best, o);
                const int oa = __shfl_xor_sync(0xffffffffu, at, o);
                if (ov > best || (ov == best && oa < at)) best = ov, at = oa;
            }
            if (lane == 0 && at < p.n_groups) gt[at] = -INFINITY;   // kept
            __syncwarp();
        }
        for (int e = lane; e < E; e += 32)
            if (gt[e / per] != -INFINITY) zt[e] = -INFINITY;
        __syncwarp();
    }
    for (int k = 0; k < top; ++k) {
        float best = -INFINITY;
        int at = 0x7fffffff;
        for (int e = lane; e < E; e += 32) {
            const float v = zt[e];
            if (v > best) best = v, at = e;     // ascending e: the first of equal values stays
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, best, o);
            const int oa = __shfl_xor_sync(0xffffffffu, at, o);
            if (ov > best || (ov == best && oa < at)) best = ov, at = oa;
        }
        if (at >= E) at = 0;     // nothing compares above -inf: the row holds NaNs
        chosen[k] = p.score_mode == 2 && p.choice_bias ? zl[at] : best;
        if (lane == 0) {
            idx[k] = at;
            zt[at] = -INFINITY;
        }
        __syncwarp();
    }
    if (lane == 0 && p.score_mode == 1) {
        for (int k = 0; k < top; ++k) wts[k] = chosen[k] * p.weight_scale;   // the scores themselves, not renormalised
    } else if (lane == 0 && p.score_mode == 2) {
        float total = 0.f;
        for (int k = 0; k < top; ++k) {
            chosen[k] = expf(chosen[k] - z_max) / z_sum;
            total += chosen[k];
        }
        const float f = p.renormalise ? p.weight_scale / (total + 1e-20f) : p.weight_scale;
        for (int k = 0; k < top; ++k) wts[k] = chosen[k] * f;
    } else if (lane == 0) {
        const float largest = chosen[0];   // the first chosen is the largest
        float sum = 0.f;
        for (int k = 0; k < top; ++k) {
            chosen[k] = expf(chosen[k] - largest);
            sum += chosen[k];
        }
        for (int k = 0; k < top; ++k) wts[k] = chosen[k] / sum;
    }
}

// A CTA routes TPB tokens: their rows wait in shared memory as 32-bit values while each warp walks the router's rows (and
// the shared expert's mixing row), one row at a time against all TPB tokens, so a row of the router is read once per CTA.
// A token's sums are made the same way whatever TPB is: lane-strided partial sums of four-wide pieces, then a shuffle tree.
template <typename TA, int TPB>
__global__ void __launch_bounds__(ROUTE_BLOCK) moe_route_kernel(const TA* __restrict__ x, int64_t ldx, int n_tokens, int d,
                                                               const float* __restrict__ wr, const float* __restrict__ br, int E, int top,
                                                               const float* __restrict__ wg, int* __restrict__ idx, float* __restrict__ wts,
                                                               float* __restrict__ gate, int vec, int score_mode, int n_groups, int keep,
                                                               int group_top, float weight_scale, const float* __restrict__ choice_bias,
                                                               int renormalise) {
    pdl_wait();
    pdl_launch_dependents();
    extern __shared__ __align__(16) float sm[];   // x [TPB][d4], then z [TPB][E], then the groups' scores [TPB][n_groups], then the choice scores [TPB][E] if they are biased
    const int d4 = (d + 3) & ~3;
    float* xs = sm;
    float* z = sm + (size_t)TPB * d4;
    float* gsc = z + (size_t)TPB * E;
    float* csc = gsc + (size_t)TPB * n_groups;
    const int t0 = blockIdx.x * TPB, nt = min(TPB, n_tokens - t0);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    for (int e = tid; e < TPB * d4; e += ROUTE_BLOCK) {
        const int tk = e / d4, i = e % d4;
        xs[e] = (tk < nt && i < d) ? to_float(x[(int64_t)(t0 + tk) * ldx + i]) : 0.f;
    }
    __syncthreads();
    for (int e = warp; e < E + (wg ? 1 : 0); e += ROUTE_BLOCK / 32) {
        const float* w = e < E ? wr + (int64_t)e * d : wg;
        float acc[TPB];
#pragma unroll
        for (int tk = 0; tk < TPB; ++tk) acc[tk] = 0.f;
        if (vec) {
#pragma unroll 4
            for (int i = lane * 4; i < d; i += 128) {
                const float4 wv = *reinterpret_cast<const float4*>(w + i);
#pragma unroll
                for (int tk = 0; tk < TPB; ++tk) {
                    const float4 xv = *reinterpret_cast<const float4*>(xs + tk * d4 + i);
                    acc[tk] = fmaf(xv.x, wv.x, acc[tk]);
                    acc[tk] = fmaf(xv.y, wv.y, acc[tk]);
                    acc[tk] = fmaf(xv.z, wv.z, acc[tk]);
                    acc[tk] = fmaf(xv.w, wv.w, acc[tk]);
                }
            }
        } else {
            for (int i = lane; i < d; i += 32) {
                const float wv = w[i];
#pragma unroll
                for (int tk = 0; tk < TPB; ++tk) acc[tk] = fmaf(xs[tk * d4 + i], wv, acc[tk]);
            }
        }
#pragma unroll
        for (int tk = 0; tk < TPB; ++tk) {
            const float sum = warp_sum(acc[tk]);
            if (lane == 0 && tk < nt) {
                if (e < E) {
                    const float logit = sum + (br ? br[e] : 0.f);
                    z[tk * E + e] = score_mode == 1 ? 1.f / (1.f + expf(-logit)) : logit;
                } else {
                    gate[t0 + tk] = 1.f / (1.f + expf(-sum));
                }
            }
        }
    }
    __syncthreads();
    // a warp per token
    const RouteRule rule{E, top, score_mode, n_groups, keep, group_top, weight_scale, choice_bias, renormalise};
    for (int tk = warp; tk < nt; tk += ROUTE_BLOCK / 32)
        choose_experts(rule, z + tk * E, gsc + tk * n_groups, csc + tk * E, lane, idx + (int64_t)(t0 + tk) * top, wts + (int64_t)(t0 + tk) * top);
}

constexpr int SORT_BLOCK = 1024, SORT_WARPS = SORT_BLOCK / 32;

// By one CTA of SORT_BLOCK threads.  seg[e] .. seg[e + 1]: expert e's rows of the list; row_token[r]: the token of row r;
// pair_row[p]: the row of pair p = t * top + k, -1 for a choice beyond the E experts.  Within an expert the rows follow the pair
// index, so the list is the same for the same routing.  A warp owns a run of consecutive pairs: it counts its experts, the counts
// become every warp's first row of every expert, and it walks its pairs again.  cnt: SORT_WARPS * E + SORT_WARPS ints in shared memory.
__device__ __forceinline__ void sort_pairs(const int* idx, int n_pairs, int top, int E, int* cnt, int* __restrict__ seg, int* __restrict__ row_token,
                                           int* __restrict__ pair_row) {
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    int* mine = cnt + warp * E;
    int* warp_total = cnt + SORT_WARPS * E;
    for (int e = tid; e < SORT_WARPS * E; e += SORT_BLOCK) cnt[e] = 0;
    __syncthreads();
    const int run = ((n_pairs + SORT_WARPS - 1) / SORT_WARPS + 31) & ~31;
    const int p_begin = min(n_pairs, warp * run), p_end = min(n_pairs, p_begin + run);
    for (int p0 = p_begin; p0 < p_end; p0 += 32) {
        const int p = p0 + lane;
        const int e = p < p_end ? idx[p] : -1;
        const bool listed = e >= 0 && e < E;
        const unsigned same = __match_any_sync(0xffffffffu, listed ? e : -1);
        if (listed && lane == __ffs(same) - 1) mine[e] += __popc(same);
        __syncwarp();
    }
    __syncthreads();
    // thread e: the warps' counts of expert e become offsets within it, then a scan over the experts
    int total = 0;
    if (tid < E)
        for (int w = 0; w < SORT_WARPS; ++w) {
            const int c = cnt[w * E + tid];
            cnt[w * E + tid] = total;
            total += c;
        }
    int incl = total;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const int v = __shfl_up_sync(0xffffffffu, incl, o);
        if (lane >= o) incl += v;
    }
    if (lane == 31) warp_total[warp] = incl;
    __syncthreads();
    int before = 0;
    for (int w = 0; w < warp; ++w) before += warp_total[w];
    const int first = before + incl - total;
    if (tid < E) {
        seg[tid] = first;
        if (tid == E - 1) seg[E] = first + total;
        for (int w = 0; w < SORT_WARPS; ++w) cnt[w * E + tid] += first;
    }
    __syncthreads();
    for (int p0 = p_begin; p0 < p_end; p0 += 32) {
        const int p = p0 + lane;
        const int e = p < p_end ? idx[p] : -1;
        const bool listed = e >= 0 && e < E;
        const unsigned same = __match_any_sync(0xffffffffu, listed ? e : -1);
        if (listed) {
            const int r = mine[e] + __popc(same & ((1u << lane) - 1u));
            row_token[r] = p / top;
            pair_row[p] = r;
        } else if (p < p_end) {
            pair_row[p] = -1;     // an identity expert: no row of the list
        }
        __syncwarp();
        if (listed && lane == __ffs(same) - 1) mine[e] += __popc(same);
        __syncwarp();
    }
}

__global__ void __launch_bounds__(SORT_BLOCK) moe_sort_kernel(const int* __restrict__ idx, int n_pairs, int top, int E, int* __restrict__ seg,
                                                              int* __restrict__ row_token, int* __restrict__ pair_row) {
    pdl_wait();
    pdl_launch_dependents();
    extern __shared__ int cnt[];
    sort_pairs(idx, n_pairs, top, E, cnt, seg, row_token, pair_row);
}

// The choice from logits that a product has made: row t of z (rows ldz apart) holds the router's R logits and, with `gate`, the
// shared expert's mixing logit behind them; with n_splits > 0 z is the product's unsummed parts, part_stride floats apart, added in
// order.  A warp per token; br: the router's bias or null.  SORT: one CTA for all tokens, which then makes the list (few tokens).
template <bool SORT>
__global__ void __launch_bounds__(SORT ? SORT_BLOCK : 256) moe_choose_kernel(const float* __restrict__ z, int64_t ldz, int n_splits, int64_t part_stride,
                                                                            int n_tokens, const float* __restrict__ br, const RouteRule rule,
                                                                            int* __restrict__ idx, float* __restrict__ wts, float* __restrict__ gate, int E,
                                                                            int* __restrict__ seg, int* __restrict__ row_token, int* __restrict__ pair_row) {
    pdl_wait();
    pdl_launch_dependents();
    extern __shared__ __align__(16) float sm[];   // a warp's logits [R], groups [n_groups] and biased scores [R]; with SORT idx and counts behind
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    const int R = rule.E, per = R * (rule.choice_bias ? 2 : 1) + rule.n_groups;
    float* zt = sm + (size_t)warp * per;
    float* gt = zt + R;
    float* cs = gt + rule.n_groups;
    int* sidx = reinterpret_cast<int*>(sm + (size_t)n_warps * per);
    auto logit = [&](int t, int e) {
        const float* p = z + (int64_t)t * ldz + e;
        float v = *p;
        for (int s = 1; s < n_splits; ++s) v += p[(int64_t)s * part_stride];
        return v;
    };
    for (int t = SORT ? warp : blockIdx.x * n_warps + warp; t < (SORT ? n_tokens : min(n_tokens, (int)(blockIdx.x + 1) * n_warps)); t += n_warps) {
        for (int e = lane; e < R; e += 32) {
            const float v = logit(t, e) + (br ? br[e] : 0.f);
            zt[e] = rule.score_mode == 1 ? 1.f / (1.f + expf(-v)) : v;
        }
        if (gate && lane == 0) gate[t] = 1.f / (1.f + expf(-logit(t, R)));
        __syncwarp();
        choose_experts(rule, zt, gt, cs, lane, SORT ? sidx + t * rule.top : idx + (int64_t)t * rule.top, wts + (int64_t)t * rule.top);
        __syncwarp();
    }
    if (SORT) {
        __syncthreads();
        sort_pairs(sidx, n_tokens * rule.top, rule.top, E, sidx + n_tokens * rule.top, seg, row_token, pair_row);
    }
}

template <typename TA>
__global__ void moe_combine_kernel(TA* __restrict__ out, const TA* __restrict__ y, const int* __restrict__ pair_row, const float* __restrict__ wts,
                                   int top, const TA* __restrict__ shared, const float* __restrict__ gate, const TA* __restrict__ input,
                                   int64_t input_ld, int d) {
    pdl_wait();
    pdl_launch_dependents();
    const int64_t t = blockIdx.x;
    const float gt = gate ? gate[t] : 1.f;
    if ((d & 3) == 0 && (input_ld & 3) == 0) {
        // four columns a thread (rows start on 8 or 16 bytes: dense [*, d] with d a multiple of 4)
        for (int i = threadIdx.x * 4; i < d; i += blockDim.x * 4) {
            float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
            for (int k = 0; k < top; ++k) {
                const float wk = wts[t * top + k];
                const int row = pair_row[t * top + k];
                const float4 v = Vec4<TA>::load(row >= 0 ? y + (int64_t)row * d + i : input + t * input_ld + i);
                acc.x = fmaf(wk, v.x, acc.x), acc.y = fmaf(wk, v.y, acc.y), acc.z = fmaf(wk, v.z, acc.z), acc.w = fmaf(wk, v.w, acc.w);
            }
            if (shared) {
                const float4 v = Vec4<TA>::load(shared + t * d + i);
                acc.x = fmaf(gt, v.x, acc.x), acc.y = fmaf(gt, v.y, acc.y), acc.z = fmaf(gt, v.z, acc.z), acc.w = fmaf(gt, v.w, acc.w);
            }
            Vec4<TA>::store(out + t * d + i, acc);
        }
        return;
    }
    for (int i = threadIdx.x; i < d; i += blockDim.x) {
        float acc = 0.f;
        for (int k = 0; k < top; ++k) {
            const int row = pair_row[t * top + k];
            acc = fmaf(wts[t * top + k], to_float(row >= 0 ? y[(int64_t)row * d + i] : input[t * input_ld + i]), acc);
        }
        if (shared) acc = fmaf(gt, to_float(shared[t * d + i]), acc);
        out[t * d + i] = from_float<TA>(acc);
    }
}

// dst[r] = src[idx[r]]: rows of d values, 16 bytes a thread where the rows allow it.
template <typename TA>
__global__ void gather_rows_kernel(TA* __restrict__ dst, const TA* __restrict__ src, int64_t ld, const int* __restrict__ idx, int d, int vec) {
    pdl_wait();
    pdl_launch_dependents();
    const int64_t r = blockIdx.x;
    const TA* from = src + (int64_t)idx[r] * ld;
    TA* to = dst + r * d;
    if (vec) {
        constexpr int PER = 16 / (int)sizeof(TA);
        for (int i = threadIdx.x * PER; i < d; i += blockDim.x * PER) *reinterpret_cast<uint4*>(to + i) = *reinterpret_cast<const uint4*>(from + i);
    } else {
        for (int i = threadIdx.x; i < d; i += blockDim.x) to[i] = from[i];
    }
}

}  // namespace

IMP_API int imp_gather_rows(void* dst, const void* src, int64_t ld, const int* idx, int n_rows, int d, int dtype, void* stream) {
    if (n_rows == 0) return 0;
    IMP_CHECK_ARG(dst && src && idx && d > 0, "imp_gather_rows: bad argument");
    const int el = dtype == IMP_F32 ? 4 : 2;
    const int vec = ((int64_t)d * el % 16 == 0 && ld * el % 16 == 0 && (uintptr_t)dst % 16 == 0 && (uintptr_t)src % 16 == 0) ? 1 : 0;
    cudaStream_t s = (cudaStream_t)stream;
    cudaError_t e = dtype == IMP_F32 ? imp_launch(gather_rows_kernel<float>, dim3(n_rows), dim3(128), 0, s, (float*)dst, (const float*)src, ld, idx, d, vec)
                                     : imp_launch(gather_rows_kernel<__nv_bfloat16>, dim3(n_rows), dim3(128), 0, s, (__nv_bfloat16*)dst,
                                                  (const __nv_bfloat16*)src, ld, idx, d, vec);
    if (e != cudaSuccess) {
        imp_set_error("imp_gather_rows: %s", cudaGetErrorString(e));
        return (int)e;
    }
    return 0;
}

template <typename TA, int TPB>
static cudaError_t launch_route(const void* x, int64_t ldx, int n_tokens, int d, const float* wr, const float* br, int E, int top, const float* wg,
                                int* idx, float* wts, float* gate, int vec, int score_mode, int n_groups, int keep, int group_top, float weight_scale, const float* choice_bias, int renormalise, size_t smem,
                                cudaStream_t s) {
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(moe_route_kernel<TA, TPB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
    }
    return imp_launch(moe_route_kernel<TA, TPB>, dim3((n_tokens + TPB - 1) / TPB), dim3(ROUTE_BLOCK), smem, s, (const TA*)x, ldx, n_tokens, d, wr, br,
                      E, top, wg, idx, wts, gate, vec, score_mode, n_groups, keep, group_top, weight_scale, choice_bias, renormalise);
}

template <typename TA>
static cudaError_t route_by_size(const void* x, int64_t ldx, int n_tokens, int d, const float* wr, const float* br, int E, int top, const float* wg,
                                 int* idx, float* wts, float* gate, int vec, int score_mode, int n_groups, int keep, int group_top, float weight_scale,
                                 const float* choice_bias, int renormalise, cudaStream_t s) {
    // more tokens a CTA where there are many (a row of the router is read once per CTA), one where there are few (more CTAs)
    int tpb = n_tokens >= 1024 ? 8 : n_tokens >= 256 ? 4 : n_tokens >= 64 ? 2 : 1;
    const int d4 = (d + 3) & ~3;
    auto bytes = [&](int t) { return ((size_t)t * d4 + (size_t)t * E * (choice_bias ? 2 : 1) + (size_t)t * n_groups) * 4; };
    while (tpb > 1 && bytes(tpb) > 160 * 1024) tpb /= 2;
    if (bytes(tpb) > 200 * 1024) return cudaErrorInvalidValue;
    switch (tpb) {
        case 8: return launch_route<TA, 8>(x, ldx, n_tokens, d, wr, br, E, top, wg, idx, wts, gate, vec, score_mode, n_groups, keep, group_top, weight_scale, choice_bias, renormalise, bytes(8), s);
        case 4: return launch_route<TA, 4>(x, ldx, n_tokens, d, wr, br, E, top, wg, idx, wts, gate, vec, score_mode, n_groups, keep, group_top, weight_scale, choice_bias, renormalise, bytes(4), s);
        case 2: return launch_route<TA, 2>(x, ldx, n_tokens, d, wr, br, E, top, wg, idx, wts, gate, vec, score_mode, n_groups, keep, group_top, weight_scale, choice_bias, renormalise, bytes(2), s);
        default: return launch_route<TA, 1>(x, ldx, n_tokens, d, wr, br, E, top, wg, idx, wts, gate, vec, score_mode, n_groups, keep, group_top, weight_scale, choice_bias, renormalise, bytes(1), s);
    }
}

// x [T, d] (activation type, rows ldx apart); wr float32 [E, d], br float32 [E] or null; wg float32 [d] or null (then
// gate is not written).  idx int32 [T, top], wts float32 [T, top], gate float32 [T].
// score_mode 0: weights are the softmax over the chosen logits; 1: scores are sigmoid(z) and a weight is its score times
// weight_scale; 2: scores are the softmax over all experts, a weight as in 1.
// choice_bias float32 [E] (or null) is added to the scores for the choice only; renormalise: the weights over their sum + 1e-20.
// group_top: how many of its largest scores a group counts by (1 or 2).  n_groups > 0: only experts of the `keep` best of n_groups equal groups of neighbours can be chosen.
IMP_API int imp_moe_route_ex(const void* x, int64_t ldx, int n_tokens, int d, const float* wr, const float* br, int E, int top, const float* wg,
                             int* idx, float* wts, float* gate, int score_mode, int n_groups, int keep, int group_top, float weight_scale,
                             const float* choice_bias, int renormalise, int act_dtype, void* stream) {
    if (n_tokens == 0) return 0;
    IMP_CHECK_ARG(x && wr && idx && wts && d > 0 && (!wg || gate), "imp_moe_route: bad argument");
    IMP_CHECK_ARG(E > 0 && E <= ROUTE_MAX_E && top > 0 && top <= E && top <= ROUTE_MAX_TOP,
                  "imp_moe_route: %d experts (at most %d), %d chosen (at most %d and no more than there are)", E, ROUTE_MAX_E, top, ROUTE_MAX_TOP);
    IMP_CHECK_ARG(score_mode >= 0 && score_mode <= 2 && (group_top == 1 || group_top == 2) && n_groups >= 0 && (n_groups == 0 || (E % n_groups == 0 && keep > 0 && keep <= n_groups &&
                                                                                             top <= keep * (E / n_groups))),
                  "imp_moe_route: %d groups over %d experts, %d kept, %d chosen", n_groups, E, keep, top);
    IMP_CHECK_ARG((!choice_bias && !renormalise) || (score_mode == 2 && n_groups == 0),
                  "imp_moe_route: a bias on the choice and renormalised weights go with softmax scores over all experts without groups");
    IMP_CHECK_ARG(score_mode != 2 || n_groups == 0 || group_top == 1, "imp_moe_route: with softmax scores over all experts groups count by their largest score");
    const int vec = (d % 4 == 0 && (uintptr_t)wr % 16 == 0 && (!wg || (uintptr_t)wg % 16 == 0)) ? 1 : 0;
    cudaStream_t s = (cudaStream_t)stream;
    cudaError_t e = act_dtype == IMP_F32 ? route_by_size<float>(x, ldx, n_tokens, d, wr, br, E, top, wg, idx, wts, gate, vec, score_mode, n_groups, keep, group_top, weight_scale, choice_bias, renormalise, s)
                                         : route_by_size<__nv_bfloat16>(x, ldx, n_tokens, d, wr, br, E, top, wg, idx, wts, gate, vec, score_mode, n_groups, keep, group_top, weight_scale, choice_bias, renormalise, s);
    if (e != cudaSuccess) {
        imp_set_error("imp_moe_route: %s (rows of %d values, %d experts)", cudaGetErrorString(e), d, E);
        return (int)e;
    }
    return 0;
}

IMP_API int imp_moe_route(const void* x, int64_t ldx, int n_tokens, int d, const float* wr, const float* br, int E, int top, const float* wg,
                          int* idx, float* wts, float* gate, int act_dtype, void* stream) {
    return imp_moe_route_ex(x, ldx, n_tokens, d, wr, br, E, top, wg, idx, wts, gate, 0, 0, 0, 2, 1.f, nullptr, 0, act_dtype, stream);
}

IMP_API int imp_moe_sort(const int* idx, int n_tokens, int top, int E, int* seg, int* row_token, int* pair_row, void* stream) {
    if (n_tokens == 0) return 0;
    IMP_CHECK_ARG(idx && seg && row_token && pair_row && top > 0 && E > 0 && E <= ROUTE_MAX_E, "imp_moe_sort: bad argument");
    const size_t smem = (size_t)(SORT_WARPS * E + SORT_WARPS) * 4;
    cudaError_t e = cudaSuccess;
    if (smem > 48 * 1024) e = cudaFuncSetAttribute(moe_sort_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e == cudaSuccess)
        e = imp_launch(moe_sort_kernel, dim3(1), dim3(SORT_BLOCK), smem, (cudaStream_t)stream, idx, n_tokens * top, top, E, seg, row_token, pair_row);
    if (e != cudaSuccess) {
        imp_set_error("imp_moe_sort: %s", cudaGetErrorString(e));
        return (int)e;
    }
    return 0;
}

// The choice of T tokens from a product's float32 logits (see moe_choose_kernel; the rule as for imp_moe_route_ex, R router outputs of
// which the first E have matrices), and the list of imp_moe_sort.  gate float32 [T] or null.  sorts: whether one kernel does both.
IMP_API int imp_moe_choose_sorts(int n_tokens, int R, int E, int top, int n_groups, int biased) {
    if (n_tokens <= 0 || n_tokens > 128) return 0;
    return ((size_t)SORT_WARPS * (R * (biased ? 2 : 1) + n_groups) + (size_t)n_tokens * top + (size_t)SORT_WARPS * (E + 1)) * 4 <= 200 * 1024 ? 1 : 0;
}
IMP_API int imp_moe_choose(const float* z, int64_t ldz, int n_splits, int64_t part_stride, int n_tokens, const float* br, int R, int E, int top, int* idx,
                           float* wts, float* gate, int score_mode, int n_groups, int keep, int group_top, float weight_scale, const float* choice_bias,
                           int renormalise, int* seg, int* row_token, int* pair_row, void* stream) {
    if (n_tokens == 0) return 0;
    IMP_CHECK_ARG(z && idx && wts && seg && row_token && pair_row && n_splits >= 0, "imp_moe_choose: bad argument");
    IMP_CHECK_ARG(R > 0 && R <= ROUTE_MAX_E && E > 0 && E <= R && top > 0 && top <= R && top <= ROUTE_MAX_TOP && ldz >= R + (gate ? 1 : 0),
                  "imp_moe_choose: %d router outputs (at most %d), %d chosen (at most %d)", R, ROUTE_MAX_E, top, ROUTE_MAX_TOP);
    IMP_CHECK_ARG(n_groups == 0 || (R % n_groups == 0 && keep > 0 && keep <= n_groups && top <= keep * (R / n_groups)), "imp_moe_choose: bad groups");
    cudaStream_t s = (cudaStream_t)stream;
    const RouteRule rule{R, top, score_mode, n_groups, keep, group_top, weight_scale, choice_bias, renormalise};
    const size_t per = ((size_t)R * (choice_bias ? 2 : 1) + n_groups) * 4;
    cudaError_t e = cudaSuccess;
    if (imp_moe_choose_sorts(n_tokens, R, E, top, n_groups, choice_bias != nullptr)) {
        const size_t smem = SORT_WARPS * per + ((size_t)n_tokens * top + (size_t)SORT_WARPS * (E + 1)) * 4;
        if (smem > 48 * 1024) e = cudaFuncSetAttribute(moe_choose_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e == cudaSuccess)
            e = imp_launch(moe_choose_kernel<true>, dim3(1), dim3(SORT_BLOCK), smem, s, z, ldz, n_splits, part_stride, n_tokens, br, rule, idx, wts, gate, E, seg,
                           row_token, pair_row);
        if (e != cudaSuccess) {
            imp_set_error("imp_moe_choose: %s", cudaGetErrorString(e));
            return (int)e;
        }
        return 0;
    }
    const size_t smem = 8 * per;
    if (smem > 48 * 1024) e = cudaFuncSetAttribute(moe_choose_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e == cudaSuccess)
        e = imp_launch(moe_choose_kernel<false>, dim3((n_tokens + 7) / 8), dim3(256), smem, s, z, ldz, n_splits, part_stride, n_tokens, br, rule, idx, wts,
                       gate, E, seg, row_token, pair_row);
    if (e != cudaSuccess) {
        imp_set_error("imp_moe_choose: %s", cudaGetErrorString(e));
        return (int)e;
    }
    return imp_moe_sort(idx, n_tokens, top, E, seg, row_token, pair_row, stream);
}

// out [T, d] = sum_k wts[t, k] * y[pair_row[t * top + k]] (+ gate[t] * shared[t]); y [T * top, d], all dense.  A negative place
// stands for row t of `input` (rows input_ld apart; needed only where identity experts can be chosen).
IMP_API int imp_moe_combine(void* out, const void* y, const int* pair_row, const float* wts, int n_tokens, int top, const void* shared,
                            const float* gate, const void* input, int64_t input_ld, int d, int act_dtype, void* stream) {
    if (n_tokens == 0) return 0;
    IMP_CHECK_ARG(out && y && pair_row && wts && top > 0 && d > 0, "imp_moe_combine: bad argument");
    cudaStream_t s = (cudaStream_t)stream;
    cudaError_t e = act_dtype == IMP_F32 ? imp_launch(moe_combine_kernel<float>, dim3(n_tokens), dim3(256), 0, s, (float*)out, (const float*)y,
                                                      pair_row, wts, top, (const float*)shared, gate, (const float*)input, input_ld, d)
                                         : imp_launch(moe_combine_kernel<__nv_bfloat16>, dim3(n_tokens), dim3(256), 0, s, (__nv_bfloat16*)out,
                                                      (const __nv_bfloat16*)y, pair_row, wts, top, (const __nv_bfloat16*)shared, gate, (const __nv_bfloat16*)input,
                                                      input_ld, d);
    if (e != cudaSuccess) {
        imp_set_error("imp_moe_combine: %s", cudaGetErrorString(e));
        return (int)e;
    }
    return 0;
}
