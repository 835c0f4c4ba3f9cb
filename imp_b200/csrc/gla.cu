// Gated linear attention: a recurrent token mixer with one matrix state S [D, Dv] per head and a decay per key channel.
//
//   alpha = sigmoid(z)^(1/tau),  z = W_a2 low + bias      (low: the inner vector of a low-rank projection)
//   S <- diag(alpha) S + k v^T;   o = S^T (q_scale q);   y = o / rms(o) per head * w * silu(gate)
//
// Everything after the projections is 32-bit arithmetic on 32-bit state whatever the activation type.  Nothing is removed from the
// state, so a token's write does not wait for a sum over the key dimension (as it does in the delta rules of delta_rule.cu): the
// only chain from token to token is one multiply-add per element, and the scan is laid out for throughput.
//
//   gla_decay    alpha for every token and channel, a thread per channel
//   gla_scan     the recurrence over portions: a CTA owns 32 value columns of one head of one sequence.  Four warps walk the
//                tokens: a thread owns four columns of D / 16 key rows in registers, as pairs for the two-wide multiply-add.  Four
//                more feed them: q, k and v from the projection's rows as they are (fetched two chunks ahead, through registers),
//                alpha through cp.async, and they carry the read-outs of the chunk before away
//   gla_decode   a step of single tokens in one kernel, from the projection's rows to y
//
// A token's arithmetic (gla_token) is the same in both, its order fixed by the sizes alone: cutting a prompt into portions or
// decoding it changes no bit.
#include <algorithm>

#include "common.cuh"

namespace {

constexpr int GLA_LANES = 16;                                   // lanes that share a column
constexpr int GLA_CT = 4;                                       // columns of a thread
constexpr int GLA_COLS = 32;                                    // columns of a block of 128 threads
constexpr int GLA_BLOCK = GLA_COLS / GLA_CT * GLA_LANES;        // 128
constexpr int GLA_MAX_D = 256;
typedef unsigned long long f32x2;

// Key rows of a lane, DPL of them (16 DPL >= D): runs of four, run j starting at 64 j + 4 lane (DPL 2: the pair at 2 lane), so that
// the lanes' 16-byte reads of a vector lie side by side.
__host__ __device__ constexpr int gla_dims(int dpl) { return GLA_LANES * dpl; }

__device__ __forceinline__ f32x2 pair_of(float lo, float hi) {
    f32x2 d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
    return d;
}
__device__ __forceinline__ float2 halves_of(f32x2 v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
    f32x2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}

// A lane's part of a vector of gla_dims(DPL) floats in shared memory.
template <int DPL>
__device__ __forceinline__ void lane_part(f32x2 (&out)[DPL / 2], const float* vec, int r) {
    if constexpr (DPL == 2) {
        out[0] = *reinterpret_cast<const f32x2*>(vec + 2 * r);
    } else {
#pragma unroll
        for (int j = 0; j < DPL / 4; ++j) {
            const ulonglong2 u = *reinterpret_cast<const ulonglong2*>(vec + 64 * j + 4 * r);
            out[2 * j] = u.x;
            out[2 * j + 1] = u.y;
        }
    }
}

// What a lane needs of a token: its parts of k, q and alpha, and its columns' values.
template <int DPL> struct TokenPart {
    f32x2 k[DPL / 2], q[DPL / 2], w[DPL / 2];
    float4 v;
    __device__ __forceinline__ void load(const float* k_vec, const float* q_vec, const float* w_vec, const float* v_cols, int r) {
        lane_part<DPL>(k, k_vec, r);
        lane_part<DPL>(w, w_vec, r);
        v = *reinterpret_cast<const float4*>(v_cols);
        lane_part<DPL>(q, q_vec, r);
    }
};

// One token: the lane's rows of its four columns decay and collect k v, then meet q; o: the lane's part of the four read-outs.
template <int DPL>
__device__ __forceinline__ void gla_token(float (&o)[GLA_CT], f32x2 (&s)[GLA_CT][DPL / 2], const TokenPart<DPL>& in) {
    const float vs[GLA_CT] = {in.v.x, in.v.y, in.v.z, in.v.w};
    f32x2 acc[GLA_CT];
#pragma unroll
    for (int p = 0; p < DPL / 2; ++p)
#pragma unroll
        for (int c = 0; c < GLA_CT; ++c) {
            s[c][p] = fma2(in.w[p], s[c][p], mul2(in.k[p], pair_of(vs[c], vs[c])));
            acc[c] = fma2(in.q[p], s[c][p], p == 0 ? 0ull : acc[c]);
        }
#pragma unroll
    for (int c = 0; c < GLA_CT; ++c) {
        const float2 h = halves_of(acc[c]);
        o[c] = h.x + h.y;
    }
}

// The sums of the read-outs' parts over the 16 lanes, in rounds of lanes 8, 4, 2, 1 apart; a lane keeps half of what it holds in
// every round that it can.  Of four columns a lane ends with column gla_column(r); of four tokens it ends with token r & 3
// (gla_reduce4), of one token every four lanes hold the same number (gla_reduce1).  The order of the additions is the same.
__device__ __forceinline__ int gla_column(int r) { return ((r >> 3) & 1) * 2 + ((r >> 2) & 1); }
__device__ __forceinline__ float keep_half(float mine_lo, float mine_hi, bool hi, int apart) {
    return (hi ? mine_hi : mine_lo) + __shfl_xor_sync(0xffffffffu, hi ? mine_lo : mine_hi, apart);
}
__device__ __forceinline__ float gla_reduce_columns(const float (&o)[GLA_CT], int r) {
    const float a0 = keep_half(o[0], o[2], r & 8, 8), a1 = keep_half(o[1], o[3], r & 8, 8);
    return keep_half(a0, a1, r & 4, 4);
}
__device__ __forceinline__ float gla_reduce1(const float (&o)[GLA_CT], int r) {
    float x = gla_reduce_columns(o, r);
    x += __shfl_xor_sync(0xffffffffu, x, 2);
    return x + __shfl_xor_sync(0xffffffffu, x, 1);
}
__device__ __forceinline__ float gla_reduce4(const float (&o)[4][GLA_CT], int r) {
    float x[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) x[u] = gla_reduce_columns(o[u], r);
    const float y0 = keep_half(x[0], x[2], r & 2, 2), y1 = keep_half(x[1], x[3], r & 2, 2);
    return keep_half(y0, y1, r & 1, 1);
}

// The state of a (slot, head, block of 32 columns): plane p of 2 DPL planes holds, for each of the 128 threads, two 32-bit pairs
// side by side (16 bytes); a warp so moves 512 contiguous bytes a plane.  Rows beyond D and columns beyond Dv stay zero.
template <int DPL>
__device__ __forceinline__ void load_state(f32x2 (&s)[GLA_CT][DPL / 2], const float* base, int tid) {
    const ulonglong2* S = reinterpret_cast<const ulonglong2*>(base);
#pragma unroll
    for (int e = 0; e < GLA_CT * DPL / 4; ++e) {
        const ulonglong2 u = S[e * GLA_BLOCK + tid];
        s[(2 * e) / (DPL / 2)][(2 * e) % (DPL / 2)] = u.x;
        s[(2 * e + 1) / (DPL / 2)][(2 * e + 1) % (DPL / 2)] = u.y;
    }
}
template <int DPL>
__device__ __forceinline__ void store_state(const f32x2 (&s)[GLA_CT][DPL / 2], float* base, int tid) {
    ulonglong2* S = reinterpret_cast<ulonglong2*>(base);
#pragma unroll
    for (int e = 0; e < GLA_CT * DPL / 4; ++e) {
        ulonglong2 u;
        u.x = s[(2 * e) / (DPL / 2)][(2 * e) % (DPL / 2)];
        u.y = s[(2 * e + 1) / (DPL / 2)][(2 * e + 1) % (DPL / 2)];
        S[e * GLA_BLOCK + tid] = u;
    }
}

__device__ __forceinline__ float gla_alpha(float z, float inv_tau) {
    const float sp = fmaxf(-z, 0.f) + log1pf(expf(-fabsf(z)));   // softplus(-z) = -log sigmoid(z)
    return expf(-sp * inv_tau);
}
__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }

}  // namespace

namespace {

// ---------------------------------------------------------------------------------------------- decay
// alpha [T, n] (n = H * D) from low [T, R] (columns of the projection's rows) and w2t = W_a2 transposed, float32 [R, n].  A CTA
// holds GLA_TOKENS tokens of 256 channels; a column of W_a2 is read once for them.  z sums over the inner index ascending.
constexpr int GLA_TOKENS = 8;
template <typename TA>
__global__ void __launch_bounds__(256) gla_decay_kernel(float* __restrict__ alpha, const TA* __restrict__ low, int64_t ld, int n_tokens, int n, int R,
                                                        const float* __restrict__ w2t, const float* __restrict__ bias, float inv_tau) {
    pdl_wait();
    pdl_launch_dependents();
    extern __shared__ __align__(16) float gla_low[];   // [R][GLA_TOKENS]
    const int t0 = blockIdx.x * GLA_TOKENS, nt = min(GLA_TOKENS, n_tokens - t0);
    for (int e = threadIdx.x; e < R * GLA_TOKENS; e += blockDim.x) {
        const int tt = e / R, j = e - tt * R;
        gla_low[j * GLA_TOKENS + tt] = tt < nt ? to_float(low[(int64_t)(t0 + tt) * ld + j]) : 0.f;
    }
    __syncthreads();
    const int c = blockIdx.y * 256 + threadIdx.x;
    if (c >= n) return;
    float z[GLA_TOKENS];
#pragma unroll
    for (int tt = 0; tt < GLA_TOKENS; ++tt) z[tt] = 0.f;
#pragma unroll 4
    for (int j = 0; j < R; ++j) {
        const float wv = w2t[(int64_t)j * n + c];
        const float4 a = *reinterpret_cast<const float4*>(gla_low + j * GLA_TOKENS), b = *reinterpret_cast<const float4*>(gla_low + j * GLA_TOKENS + 4);
        z[0] = fmaf(a.x, wv, z[0]), z[1] = fmaf(a.y, wv, z[1]), z[2] = fmaf(a.z, wv, z[2]), z[3] = fmaf(a.w, wv, z[3]);
        z[4] = fmaf(b.x, wv, z[4]), z[5] = fmaf(b.y, wv, z[5]), z[6] = fmaf(b.z, wv, z[6]), z[7] = fmaf(b.w, wv, z[7]);
    }
    const float zb = bias[c];
#pragma unroll
    for (int tt = 0; tt < GLA_TOKENS; ++tt)
        if (tt < nt) alpha[(int64_t)(t0 + tt) * n + c] = gla_alpha(z[tt] + zb, inv_tau);
}

// ----------------------------------------------------------------------------------------------- scan
// proj rows: [q: H*D | k: H*D | v: H*Dv | ...] in the activations' type; alpha [T, H*D], out [T, H*Dv] float32.
__host__ __device__ constexpr int gla_chunk(int dpl) { return dpl <= 8 ? 16 : 8; }
template <int DPL> constexpr size_t gla_scan_smem() {
    return (size_t)(2 * gla_chunk(DPL) * (3 * gla_dims(DPL) + 2 * GLA_COLS)) * sizeof(float);
}

template <typename TA> __device__ __forceinline__ void widen16(float* dst, const uint4 u, float f) {
    if constexpr (sizeof(TA) == 4) {
        *reinterpret_cast<float4*>(dst) = make_float4(__uint_as_float(u.x) * f, __uint_as_float(u.y) * f, __uint_as_float(u.z) * f, __uint_as_float(u.w) * f);
    } else {
        const uint32_t ws[4] = {u.x, u.y, u.z, u.w};
        float v[8];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            v[2 * i] = __uint_as_float(ws[i] << 16) * f;
            v[2 * i + 1] = __uint_as_float(ws[i] & 0xffff0000u) * f;
        }
        *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]);
        *reinterpret_cast<float4*>(dst + 4) = make_float4(v[4], v[5], v[6], v[7]);
    }
}

// VEC: D and Dv are multiples of 16 bytes' worth of activations and every row starts on 16 bytes.
template <typename TA, int DPL, bool VEC>
__global__ void __launch_bounds__(2 * GLA_BLOCK) gla_scan_kernel(const TA* __restrict__ proj, int64_t ld, const float* __restrict__ alpha, float q_scale,
                                                                 float* __restrict__ state, float* __restrict__ out, const int* __restrict__ q_start,
                                                                 const int* __restrict__ slots, int D, int H, int Dv) {
    pdl_wait();
    pdl_launch_dependents();
    constexpr int DP = gla_dims(DPL), CH = gla_chunk(DPL), PER = 16 / (int)sizeof(TA);
    constexpr int NQ = (CH * DP / PER + GLA_BLOCK - 1) / GLA_BLOCK, NV = (CH * GLA_COLS / PER + GLA_BLOCK - 1) / GLA_BLOCK;
    extern __shared__ __align__(16) float gla_smem[];
    float* q_s = gla_smem;                         // [2][CH][DP]
    float* k_s = q_s + 2 * CH * DP;
    float* w_s = k_s + 2 * CH * DP;
    float* v_s = w_s + 2 * CH * DP;                // [2][CH][GLA_COLS]
    float* o_s = v_s + 2 * CH * GLA_COLS;          // [2][CH][GLA_COLS]
    const int tid = threadIdx.x % GLA_BLOCK;
    const bool feeds = threadIdx.x >= GLA_BLOCK;
    const int col0 = blockIdx.x * GLA_COLS, h = blockIdx.y, seq = blockIdx.z;
    const int start = q_start[seq], n = q_start[seq + 1] - start;
    if (n <= 0) return;
    const int64_t HD = (int64_t)H * D, HV = (int64_t)H * Dv;
    const int n_chunks = (n + CH - 1) / CH;
    if (feeds) {
        uint4 qr[VEC ? NQ : 1], kr[VEC ? NQ : 1], vr[VEC ? NV : 1];
        // a chunk's q, k and v into registers
        auto fetch = [&](int chunk) {
            if constexpr (VEC) {
                const int t0 = chunk * CH, nt = min(CH, n - t0);
                const uint4 zero = make_uint4(0, 0, 0, 0);
#pragma unroll
                for (int e = 0; e < NQ; ++e) {
                    const int idx = tid + e * GLA_BLOCK, tt = idx / (DP / PER), d = idx % (DP / PER) * PER;
                    const bool ok = tt < nt && d < D;
                    const TA* row = proj + (int64_t)(start + t0 + (ok ? tt : 0)) * ld + (int64_t)h * D + (ok ? d : 0);
                    qr[e] = ok ? *reinterpret_cast<const uint4*>(row) : zero;
                    kr[e] = ok ? *reinterpret_cast<const uint4*>(row + HD) : zero;
                }
#pragma unroll
                for (int e = 0; e < NV; ++e) {
                    const int idx = tid + e * GLA_BLOCK, tt = idx / (GLA_COLS / PER), c = idx % (GLA_COLS / PER) * PER;
                    const bool ok = tt < nt && col0 + c < Dv;
                    vr[e] = ok ? *reinterpret_cast<const uint4*>(proj + (int64_t)(start + t0 + tt) * ld + 2 * HD + (int64_t)h * Dv + col0 + c) : zero;
                }
            }
        };
        // the chunk's q, k and v from the registers (or straight from memory) into its buffer; its alpha is asked for
        auto stash = [&](int chunk) {
            const int t0 = chunk * CH, nt = min(CH, n - t0), buf = chunk & 1;
            constexpr int W = VEC ? 4 : 1;
            for (int idx = tid; idx < CH * DP / W; idx += GLA_BLOCK) {
                const int tt = idx / (DP / W), d = idx % (DP / W) * W;
                const bool ok = tt < nt && d < D;
                const float* src = alpha + (ok ? (int64_t)(start + t0 + tt) * HD + (int64_t)h * D + d : 0);
                const uint32_t dst = (uint32_t)__cvta_generic_to_shared(w_s + buf * CH * DP + idx * W);
                if constexpr (VEC) asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(src), "r"(ok ? 16 : 0) : "memory");
                else asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;\n" ::"r"(dst), "l"(src), "r"(ok ? 4 : 0) : "memory");
            }
            if constexpr (VEC) {
#pragma unroll
                for (int e = 0; e < NQ; ++e) {
                    const int idx = tid + e * GLA_BLOCK;
                    if (NQ * GLA_BLOCK > CH * DP / PER && idx >= CH * DP / PER) break;
                    widen16<TA>(q_s + buf * CH * DP + idx * PER, qr[e], q_scale);
                    widen16<TA>(k_s + buf * CH * DP + idx * PER, kr[e], 1.f);
                }
#pragma unroll
                for (int e = 0; e < NV; ++e) {
                    const int idx = tid + e * GLA_BLOCK;
                    if (NV * GLA_BLOCK > CH * GLA_COLS / PER && idx >= CH * GLA_COLS / PER) break;
                    widen16<TA>(v_s + buf * CH * GLA_COLS + idx * PER, vr[e], 1.f);
                }
            } else {
                for (int idx = tid; idx < CH * DP; idx += GLA_BLOCK) {
                    const int tt = idx / DP, d = idx % DP;
                    const bool ok = tt < nt && d < D;
                    const TA* row = proj + (int64_t)(start + t0 + (ok ? tt : 0)) * ld + (int64_t)h * D + (ok ? d : 0);
                    q_s[buf * CH * DP + idx] = ok ? to_float(row[0]) * q_scale : 0.f;
                    k_s[buf * CH * DP + idx] = ok ? to_float(row[HD]) : 0.f;
                }
                for (int idx = tid; idx < CH * GLA_COLS; idx += GLA_BLOCK) {
                    const int tt = idx / GLA_COLS, c = idx % GLA_COLS;
                    const bool ok = tt < nt && col0 + c < Dv;
                    v_s[buf * CH * GLA_COLS + idx] = ok ? to_float(proj[(int64_t)(start + t0 + tt) * ld + 2 * HD + (int64_t)h * Dv + col0 + c]) : 0.f;
                }
            }
        };
        auto carry_away = [&](int chunk) {
            const int t0 = chunk * CH, nt = min(CH, n - t0);
            const float* ob = o_s + (chunk & 1) * CH * GLA_COLS;
            float* dst = out + (int64_t)(start + t0) * HV + (int64_t)h * Dv + col0;
#pragma unroll
            for (int e = tid; e < CH * GLA_COLS; e += GLA_BLOCK) {
                const int tt = e / GLA_COLS, c = e % GLA_COLS;
                if (tt < nt && col0 + c < Dv) dst[(int64_t)tt * HV + c] = ob[e];
            }
        };
        fetch(0);
        stash(0);
        if (n_chunks > 1) fetch(1);
        asm volatile("cp.async.wait_all;\n" ::: "memory");
        __syncthreads();
        for (int i = 0; i < n_chunks; ++i) {
            // while chunk i is walked: the next one's buffer is filled, the one after is fetched, the read-outs before leave
            if (i + 1 < n_chunks) stash(i + 1);
            if (i + 2 < n_chunks) fetch(i + 2);
            if (i > 0) carry_away(i - 1);
            asm volatile("cp.async.wait_all;\n" ::: "memory");
            __syncthreads();
        }
        carry_away(n_chunks - 1);
        return;
    }
    const int r = tid & (GLA_LANES - 1), cg = tid / GLA_LANES;
    float* S = state + (((int64_t)slots[seq] * H + h) * gridDim.x + blockIdx.x) * (GLA_COLS * DP);
    f32x2 s[GLA_CT][DPL / 2];
    load_state<DPL>(s, S, tid);
    __syncthreads();
    for (int i = 0; i < n_chunks; ++i) {
        const int nt = min(CH, n - i * CH), buf = i & 1;
        const float *kb = k_s + buf * CH * DP, *qb = q_s + buf * CH * DP, *wb = w_s + buf * CH * DP, *vb = v_s + buf * CH * GLA_COLS + cg * GLA_CT;
        const uint32_t ob = (uint32_t)__cvta_generic_to_shared(o_s + buf * CH * GLA_COLS + cg * GLA_CT + gla_column(r));
        // four tokens at a time, a token's vectors asked for while the token before it is worked on; the read-outs' stores are
        // plain instructions that name no memory, so that the compiler may move the next loads ahead of them
        TokenPart<DPL> in[2];
        in[0].load(kb, qb, wb, vb, r);
        int tt = 0;
#pragma unroll 2
        for (; tt + 4 <= nt; tt += 4) {
            float o[4][GLA_CT];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const int next = min(tt + u + 1, CH - 1);
                in[(u + 1) & 1].load(kb + next * DP, qb + next * DP, wb + next * DP, vb + next * GLA_COLS, r);
                gla_token<DPL>(o[u], s, in[u & 1]);
            }
            asm volatile("st.shared.f32 [%0], %1;" ::"r"(ob + (uint32_t)((tt + (r & 3)) * GLA_COLS * 4)), "f"(gla_reduce4(o, r)));
        }
        for (; tt < nt; ++tt) {
            float o[GLA_CT];
            in[0].load(kb + tt * DP, qb + tt * DP, wb + tt * DP, vb + tt * GLA_COLS, r);
            gla_token<DPL>(o, s, in[0]);
            const float x = gla_reduce1(o, r);
            if ((r & 3) == 0) asm volatile("st.shared.f32 [%0], %1;" ::"r"(ob + (uint32_t)(tt * GLA_COLS * 4)), "f"(x));
        }
        __syncthreads();
    }
    store_state<DPL>(s, S, tid);
}

}  // namespace

namespace {

// --------------------------------------------------------------------------------------------- decode
// A step of single tokens, from the projection's rows to the gated read-out: a CTA per (head, sequence), two groups of 128 threads
// that take blocks of 32 columns in turn.  The decay's sum, the token's arithmetic and the norm's sum have the order of the
// kernels that run for portions (gla_decay, gla_scan, gdr_output).
constexpr int GLA_DEC_BLOCK = 2 * GLA_BLOCK;
template <typename TA, int DPL>
__global__ void __launch_bounds__(GLA_DEC_BLOCK) gla_decode_kernel(const TA* __restrict__ proj, int64_t ld, int H, int D, int Dv, int R,
                                                                   const float* __restrict__ w2t, const float* __restrict__ bias, float inv_tau,
                                                                   float q_scale, const float* __restrict__ out_w, float eps, float* __restrict__ state,
                                                                   const int* __restrict__ slots, TA* __restrict__ y) {
    pdl_wait();
    pdl_launch_dependents();
    constexpr int DP = gla_dims(DPL);
    extern __shared__ __align__(16) float gla_smem[];   // o [whole blocks of columns], low [R]
    __shared__ __align__(16) float k_s[DP], q_s[DP], w_s[DP];
    const int n_blocks = (Dv + GLA_COLS - 1) / GLA_COLS;
    float* o_s = gla_smem;
    float* low_s = gla_smem + n_blocks * GLA_COLS;
    const int tid = threadIdx.x, lane = tid & 31, g = tid / GLA_BLOCK, gt = tid % GLA_BLOCK, r = gt & (GLA_LANES - 1), cg = gt / GLA_LANES;
    const int h = blockIdx.x;
    const int64_t t = blockIdx.y;
    const int64_t HD = (int64_t)H * D, HV = (int64_t)H * Dv;
    const TA* row = proj + t * ld;
    float* S0 = state + ((int64_t)slots[t] * H + h) * n_blocks * (GLA_COLS * DP);
    f32x2 s[GLA_CT][DPL / 2];
    if (g < n_blocks) load_state<DPL>(s, S0 + (int64_t)g * (GLA_COLS * DP), gt);
    for (int j = tid; j < R; j += GLA_DEC_BLOCK) low_s[j] = to_float(row[2 * HD + 2 * HV + j]);
    __syncthreads();
    if (tid < DP) {
        float qq = 0.f, kk = 0.f, ww = 0.f;
        if (tid < D) {
            qq = to_float(row[(int64_t)h * D + tid]) * q_scale;
            kk = to_float(row[HD + (int64_t)h * D + tid]);
            float z = 0.f;
            const float* col = w2t + (int64_t)h * D + tid;
#pragma unroll 8
            for (int j = 0; j < R; ++j) z = fmaf(low_s[j], col[(int64_t)j * HD], z);
            ww = gla_alpha(z + bias[(int64_t)h * D + tid], inv_tau);
        }
        q_s[tid] = qq;
        k_s[tid] = kk;
        w_s[tid] = ww;
    }
    __syncthreads();
    for (int cb = g; cb < n_blocks; cb += 2) {
        if (cb != g) load_state<DPL>(s, S0 + (int64_t)cb * (GLA_COLS * DP), gt);
        const int c0 = cb * GLA_COLS + cg * GLA_CT;
        float v[GLA_CT];
#pragma unroll
        for (int c = 0; c < GLA_CT; ++c) v[c] = c0 + c < Dv ? to_float(row[2 * HD + (int64_t)h * Dv + c0 + c]) : 0.f;
        float o[GLA_CT];
        TokenPart<DPL> in;
        lane_part<DPL>(in.k, k_s, r);
        lane_part<DPL>(in.q, q_s, r);
        lane_part<DPL>(in.w, w_s, r);
        in.v = make_float4(v[0], v[1], v[2], v[3]);
        gla_token<DPL>(o, s, in);
        const float x = gla_reduce1(o, r);
        if ((r & 3) == 0) o_s[c0 + gla_column(r)] = x;
        store_state<DPL>(s, S0 + (int64_t)cb * (GLA_COLS * DP), gt);
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = lane; c < Dv; c += 32) ss = fmaf(o_s[c], o_s[c], ss);
    ss = warp_sum(ss);
    const float inv = rsqrtf(ss / (float)Dv + eps);
    for (int c = tid; c < Dv; c += GLA_DEC_BLOCK) {
        const float gate = to_float(row[2 * HD + HV + (int64_t)h * Dv + c]);
        y[(t * H + h) * Dv + c] = from_float<TA>(o_s[c] * inv * out_w[c] * silu_f(gate));
    }
}

int gla_dims_per_lane(int D) { return D <= 32 ? 2 : D <= 64 ? 4 : D <= 128 ? 8 : 16; }

template <typename TA, int DPL, bool VEC>
cudaError_t launch_scan(dim3 grid, cudaStream_t s, const void* proj, int64_t ld, const float* alpha, float q_scale, float* state, float* out,
                        const int* q_start, const int* slots, int D, int H, int Dv) {
    constexpr size_t smem = gla_scan_smem<DPL>();
    static bool raised = false;   // per instantiation
    if (!raised && smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(gla_scan_kernel<TA, DPL, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
        raised = true;
    }
    // an ordinary dependent launch: CTAs that stay for a whole portion must not become resident while earlier kernels run
    gla_scan_kernel<TA, DPL, VEC><<<grid, 2 * GLA_BLOCK, smem, s>>>((const TA*)proj, ld, alpha, q_scale, state, out, q_start, slots, D, H, Dv);
    return cudaGetLastError();
}

}  // namespace

// Floats of one slot's state.
IMP_API int64_t imp_gla_state_floats(int H, int D, int Dv) {
    return (int64_t)H * ((Dv + GLA_COLS - 1) / GLA_COLS) * GLA_COLS * gla_dims(gla_dims_per_lane(D));
}

// alpha [n_tokens, n] = sigmoid(low w2t + bias)^(1/tau); low: n_tokens rows, ld apart, of R values in the activations' type.
IMP_API int imp_gla_decay(float* alpha, const void* low, int64_t ld, int n_tokens, int n, int R, const float* w2t, const float* bias, float tau,
                          int act_dtype, void* stream) {
    if (n_tokens == 0) return 0;
    IMP_CHECK_ARG(alpha && low && w2t && bias && n > 0 && R > 0 && ld >= R && tau > 0.f, "imp_gla_decay: bad argument");
    const size_t smem = (size_t)R * GLA_TOKENS * 4;
    IMP_CHECK_ARG(smem <= 48 * 1024, "imp_gla_decay: an inner size of %d is more than this kernel holds", R);
    cudaStream_t s = (cudaStream_t)stream;
    const dim3 grid((n_tokens + GLA_TOKENS - 1) / GLA_TOKENS, (n + 255) / 256);
    if (act_dtype == IMP_F32)
        imp_launch(gla_decay_kernel<float>, grid, dim3(256), smem, s, alpha, (const float*)low, ld, n_tokens, n, R, w2t, bias, 1.f / tau);
    else
        imp_launch(gla_decay_kernel<__nv_bfloat16>, grid, dim3(256), smem, s, alpha, (const __nv_bfloat16*)low, ld, n_tokens, n, R, w2t, bias, 1.f / tau);
    IMP_RETURN_LAUNCH();
}

// The recurrence over a step's portions: proj rows [q: H*D | k: H*D | v: H*Dv | ...], alpha [T, H*D], out [T, H*Dv] float32; state
// [slots, imp_gla_state_floats()], zero at a request's start, updated in place.
IMP_API int imp_gla_scan(const void* proj, int64_t ld, const float* alpha, float q_scale, float* state, float* out, const int* q_start, const int* slots,
                         int n_seqs, int D, int H, int Dv, int act_dtype, void* stream) {
    if (n_seqs == 0) return 0;
    IMP_CHECK_ARG(proj && alpha && state && out && q_start && slots, "imp_gla_scan: null pointer");
    IMP_CHECK_ARG(D > 0 && Dv > 0 && H > 0 && H <= 65535 && n_seqs <= 65535 && ld >= 2 * (int64_t)H * D + (int64_t)H * Dv, "imp_gla_scan: bad sizes");
    if (D > GLA_MAX_D) {
        imp_set_error("imp_gla_scan: key size %d exceeds %d", D, GLA_MAX_D);
        return IMP_ERR_UNSUPPORTED;
    }
    cudaStream_t s = (cudaStream_t)stream;
    const dim3 grid((Dv + GLA_COLS - 1) / GLA_COLS, H, n_seqs);
    const int per = act_dtype == IMP_F32 ? 4 : 8;
    const bool vec = D % per == 0 && Dv % per == 0 && ld % per == 0 && (uintptr_t)proj % 16 == 0 && (uintptr_t)alpha % 16 == 0;
    cudaError_t e;
#define GLA_SCAN_T(TA, DPL)                                                                                                \
    e = vec ? launch_scan<TA, DPL, true>(grid, s, proj, ld, alpha, q_scale, state, out, q_start, slots, D, H, Dv)          \
            : launch_scan<TA, DPL, false>(grid, s, proj, ld, alpha, q_scale, state, out, q_start, slots, D, H, Dv)
#define GLA_SCAN(DPL)                                      \
    do {                                                   \
        if (act_dtype == IMP_F32) GLA_SCAN_T(float, DPL);  \
        else GLA_SCAN_T(__nv_bfloat16, DPL);               \
    } while (0)
    switch (gla_dims_per_lane(D)) {
        case 2: GLA_SCAN(2); break;
        case 4: GLA_SCAN(4); break;
        case 8: GLA_SCAN(8); break;
        default: GLA_SCAN(16); break;
    }
#undef GLA_SCAN
#undef GLA_SCAN_T
    if (e != cudaSuccess) {
        imp_set_error("imp_gla_scan: %s", cudaGetErrorString(e));
        return (int)e;
    }
    return 0;
}

// A step of single tokens (token t belongs to sequence t): projection rows [q | k | v | gate | low: R | ...] to the gated read-out
// y [n_tokens, H * Dv], the state updated.
IMP_API int imp_gla_decode(const void* proj, int64_t ld, int n_tokens, int H, int D, int Dv, int R, const float* w2t, const float* bias, float tau,
                           float q_scale, const float* out_w, float eps, float* state, const int* slots, void* y, int act_dtype, void* stream) {
    if (n_tokens == 0) return 0;
    IMP_CHECK_ARG(proj && w2t && bias && out_w && state && slots && y, "imp_gla_decode: null pointer");
    IMP_CHECK_ARG(H > 0 && D > 0 && D <= GLA_MAX_D && Dv > 0 && R > 0 && tau > 0.f && n_tokens <= 65535 &&
                      ld >= 2 * ((int64_t)H * D + (int64_t)H * Dv) + R,
                  "imp_gla_decode: bad sizes (key size %d of at most %d)", D, GLA_MAX_D);
    const size_t smem = (size_t)((Dv + GLA_COLS - 1) / GLA_COLS * GLA_COLS + R) * 4;
    if (smem > 40 * 1024) return IMP_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
    const dim3 grid(H, n_tokens);
    cudaError_t e;
#define GLA_DECODE_T(TA, DPL)                                                                                                                      \
    e = imp_launch(gla_decode_kernel<TA, DPL>, grid, dim3(GLA_DEC_BLOCK), smem, s, (const TA*)proj, ld, H, D, Dv, R, w2t, bias, 1.f / tau, q_scale, \
                   out_w, eps, state, slots, (TA*)y)
#define GLA_DECODE(DPL)                                      \
    do {                                                     \
        if (act_dtype == IMP_F32) GLA_DECODE_T(float, DPL);  \
        else GLA_DECODE_T(__nv_bfloat16, DPL);               \
    } while (0)
    switch (gla_dims_per_lane(D)) {
        case 2: GLA_DECODE(2); break;
        case 4: GLA_DECODE(4); break;
        case 8: GLA_DECODE(8); break;
        default: GLA_DECODE(16); break;
    }
#undef GLA_DECODE
#undef GLA_DECODE_T
    if (e != cudaSuccess) {
        imp_set_error("imp_gla_decode: %s", cudaGetErrorString(e));
        return (int)e;
    }
    return 0;
}
