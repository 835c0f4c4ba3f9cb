// Between a q,k,v product and the paged attention kernels, for attention whose heads are normalised, rotated in
// part, scaled per head and whose values are normalised; and the small kernels of blocks that combine two mixers
// or gate their heads.
//
//   qkv_prepare      per token (qkv_prepare.h): a bias on q, k and v (optional); q and k heads -> RMS norm (optional, with or
//                    without a weight, before or after the rotation), rotation of the first `rot` entries (pairs i, i + rot/2,
//                    or neighbours 2i, 2i + 1; optionally times a constant); q times a number per head (optional) -> q_out,
//                    padded to the cache's head size; k -> K page; v heads -> divided by their root mean square (optional) -> V
//                    page.  Key and value heads may have different sizes: the cache's head size is the larger one, the rest
//                    of a row is zeros.  With v_share = n, n neighbouring key heads read one value head (the product holds
//                    Hkv / n of them) and each caches a copy of it.
//   diff_combine     two softmax maps per head over the same values: o = a1 - lambda * a2, o / rms(o) * out_scale
//   head_gate        y[t, h, :] *= sigmoid(g[t, h])
//   rms_pair_mean    out = ca * a / rms(a) * wa + cb * b / rms(b) * wb   (two branch outputs, each normalised over the width)
//   gated_act        out = act(gate) * up for gelu (tanh form) and silu over [gate | up] rows
//   act_rows         out[t, :] = act(x[t, c0 : c0 + n])  (a slice of a product's rows made dense, tanh or identity)
// Norm statistics, angles, the rotation and the per-head factors are 32-bit; results are rounded once.
#include "common.cuh"
#include "qkv_prepare.h"

constexpr int QP_BLOCK = 256;
constexpr int QP_WARPS = QP_BLOCK / 32;
constexpr int QP_UNITS = 16;     // units of one token a CTA takes in steps of few tokens: the token's angles are made once for all of them
constexpr int QP_MAX_D = 512;

// cos and sin of a pair's angle at a position.  The angle is made in turns, pos * turns with turns = hi + lo: the product with
// hi is exact as a float and its rounding error, whole turns leave exactly, so what reaches sincospif is right to 32-bit at any
// position (pos * angle rounded to a float would lose a digit per decade of positions).
__device__ __forceinline__ void rotation_angle(float pos, float hi, float lo, float mult, float* sn, float* cs) {
    const float whole = pos * hi, err = fmaf(pos, hi, -whole);
    sincospif(2.f * ((whole - rintf(whole)) + fmaf(pos, lo, err)), sn, cs);
    *sn *= mult;
    *cs *= mult;
}

// A CTA per (token, group of units), a warp per unit; units: Hq query heads, then Hkv key heads, then Hkv value heads; PER
// entries of a head a lane (the cache's head size is at most 32 * PER).
template <typename TA, int PER>
__global__ void __launch_bounds__(QP_BLOCK) qkv_prepare_kernel(const ImpQkvPrepare p, int units_per_cta, int* status) {
    pdl_wait();
    pdl_launch_dependents();
    __shared__ float rot_s[QP_WARPS][32 * PER];
    __shared__ float cos_s[16 * PER], sin_s[16 * PER];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int Hq = p.Hq, Hkv = p.Hkv, D = p.D, Dc = p.Dc, rot = p.rot;
    const int units = Hq + 2 * Hkv;
    const int64_t t = blockIdx.x;
    const int seq = p.seq_of_token[t], pos = p.positions[t];
    if (seq < 0 || seq >= p.n_seqs || pos < 0 || pos / p.page_size >= p.bt_stride) {
        if (threadIdx.x == 0 && blockIdx.y == 0) imp_report(status, seq < 0 || seq >= p.n_seqs ? IMP_BAD_SEQUENCE : IMP_BAD_POSITION);
        return;
    }
    const int half = rot / 2;
    const int u_begin = blockIdx.y * units_per_cta, u_end = min(units, u_begin + units_per_cta);
    if (rot > 0 && u_begin < Hq + Hkv) {     // a group of value heads rotates nothing
        for (int i = threadIdx.x; i < half; i += QP_BLOCK) rotation_angle((float)pos, p.turns[i], p.turns[half + i], p.rot_mult, &sin_s[i], &cos_s[i]);
    }
    __syncthreads();
    const int page = p.block_table[(int64_t)seq * p.bt_stride + pos / p.page_size];
    for (int unit = u_begin + warp; unit < u_end; unit += QP_WARPS) {
        const bool is_q = unit < Hq, is_v = unit >= Hq + Hkv;
        const int head = is_q ? unit : is_v ? unit - Hq - Hkv : unit - Hq;
        const int n = is_v ? p.Dv : D;
        const int64_t col = is_q ? (int64_t)head * D : is_v ? (int64_t)(Hq + Hkv) * D + (int64_t)(head / p.v_share) * p.Dv : (int64_t)(Hq + head) * D;
        const TA* src = p.parts ? nullptr : (const TA*)p.proj + t * p.ld + col;
        TA* dst;
        if (is_q) {
            dst = (TA*)p.q_out + t * p.q_ld + (int64_t)head * Dc;
        } else {
            if (page < 0 || page >= p.num_pages) {
                if (lane == 0) imp_report(status, IMP_BAD_PAGE);
                continue;
            }
            TA* cache = (TA*)(is_v ? p.v_cache : p.k_cache);
            if (!cache) continue;
            dst = cache + (((int64_t)page * Hkv + head) * p.page_size + pos % p.page_size) * Dc;   // pages are [page][kv head][slot][entry]
        }
        float x[PER];
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int d = lane + i * 32;
            x[i] = 0.f;
            if (d < n) {
                if (src) {
                    x[i] = to_float(src[d]);
                } else {
                    float acc = 0.f;
                    for (int s = 0; s < p.n_splits; ++s) acc += p.parts[((int64_t)s * p.n_tokens + t) * p.ld + col + d];
                    x[i] = to_float(from_float<TA>(acc));
                }
                if (p.bias) x[i] += p.bias[col + d];
            }
        }
        const float* nw = is_q ? p.q_norm_w : is_v ? nullptr : p.k_norm_w;
        auto norm = [&] {
            float ss = 0.f;
#pragma unroll
            for (int i = 0; i < PER; ++i) ss = fmaf(x[i], x[i], ss);     // entries beyond the head are zero
            ss = warp_sum(ss);
            const float r = rsqrtf(ss / (float)n + p.eps);
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                const int d = lane + i * 32;
                if (d < n) x[i] = x[i] * r * (nw ? nw[d] : 1.f);
            }
        };
        if (is_v ? p.v_norm != 0 : p.qk_norm == QK_NORM_BEFORE_ROTATION) norm();
        if (!is_v && rot > 0 && p.pairing == 1) {
            // neighbours: entry 2i pairs with 2i + 1, which the next lane holds
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                const int d = lane + i * 32;
                const float partner = __shfl_xor_sync(0xffffffffu, x[i], 1);
                if (d < rot) {
                    const float sn = sin_s[d >> 1], cs = cos_s[d >> 1];
                    x[i] = (d & 1) ? x[i] * cs + partner * sn : x[i] * cs - partner * sn;
                }
            }
        } else if (!is_v && rot > 0) {
            // entry d < rot/2 pairs with d + rot/2, which another lane holds: the head goes through shared memory once
            float* row = rot_s[warp];
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                const int d = lane + i * 32;
                if (d < rot) row[d] = x[i];
            }
            __syncwarp();
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                const int d = lane + i * 32;
                if (d < rot) {
                    const int fi = d < half ? d : d - half;
                    const float partner = row[d < half ? d + half : d - half];
                    const float sn = sin_s[fi], cs = cos_s[fi];
                    // (u, v) -> (u cos - v sin, v cos + u sin)
                    x[i] = d < half ? x[i] * cs - partner * sn : x[i] * cs + partner * sn;
                }
            }
            __syncwarp();     // the row is written again for the warp's next unit
        }
        if (!is_v && p.qk_norm == QK_NORM_AFTER_ROTATION) norm();
        const float mult = (is_q && p.head_mult) ? p.head_mult[head] : 1.f;
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int d = lane + i * 32;
            if (d < Dc) dst[d] = from_float<TA>(d < n ? x[i] * mult : 0.f);
        }
    }
}

// The same for 16-bit activations with eight neighbouring entries a lane (16-byte loads and stores; a rotated pair of
// neighbours is in one lane): LPH lanes a head, 32 / LPH heads a warp at once.  Head sizes that are multiples of 8 up to
// 8 * LPH, rows that start on 16 bytes, no rotation of halves.  PARTS: from the product's unsummed parts.
template <int LPH, bool PARTS>
__global__ void __launch_bounds__(QP_BLOCK) qkv_prepare_vec_kernel(const ImpQkvPrepare p, int units_per_cta, int* status) {
    pdl_wait();
    pdl_launch_dependents();
    using TA = __nv_bfloat16;
    constexpr int UPW = 32 / LPH;
    __shared__ __align__(16) float cos_s[4 * LPH], sin_s[4 * LPH];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int sub = lane / LPH, d0 = (lane % LPH) * 8;
    const int Hq = p.Hq, Hkv = p.Hkv, D = p.D, Dc = p.Dc, rot = p.rot;
    const int units = Hq + 2 * Hkv;
    const int64_t t = blockIdx.x;
    const int seq = p.seq_of_token[t], pos = p.positions[t];
    if (seq < 0 || seq >= p.n_seqs || pos < 0 || pos / p.page_size >= p.bt_stride) {
        if (threadIdx.x == 0 && blockIdx.y == 0) imp_report(status, seq < 0 || seq >= p.n_seqs ? IMP_BAD_SEQUENCE : IMP_BAD_POSITION);
        return;
    }
    const int half = rot / 2;
    const int u_begin = blockIdx.y * units_per_cta, u_end = min(units, u_begin + units_per_cta);
    if (u_begin < Hq + Hkv) {
        for (int i = threadIdx.x; i < half; i += QP_BLOCK) rotation_angle((float)pos, p.turns[i], p.turns[half + i], p.rot_mult, &sin_s[i], &cos_s[i]);
    }
    __syncthreads();
    const int page = p.block_table[(int64_t)seq * p.bt_stride + pos / p.page_size];
    const bool page_ok = page >= 0 && page < p.num_pages;
    if (!page_ok && threadIdx.x == 0 && u_end > Hq) imp_report(status, IMP_BAD_PAGE);
    for (int base = u_begin + warp * UPW; base < u_end; base += QP_WARPS * UPW) {   // the same for every lane of a warp
        const int unit = base + sub;
        const bool there = unit < u_end;
        const bool is_q = unit < Hq, is_v = unit >= Hq + Hkv;
        const int head = is_q ? unit : is_v ? unit - Hq - Hkv : unit - Hq;
        const int n = is_v ? p.Dv : D;
        const int64_t col = is_q ? (int64_t)head * D : is_v ? (int64_t)(Hq + Hkv) * D + (int64_t)(head / p.v_share) * p.Dv : (int64_t)(Hq + head) * D;
        const bool mine = there && d0 < n;
        float x[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) x[i] = 0.f;
        if (PARTS && mine) {
            const float* src = p.parts + t * p.ld + col + d0;
#pragma unroll 4
            for (int s = 0; s < p.n_splits; ++s, src += (int64_t)p.n_tokens * p.ld) {
                const float4 a = *reinterpret_cast<const float4*>(src), b = *reinterpret_cast<const float4*>(src + 4);
                x[0] += a.x, x[1] += a.y, x[2] += a.z, x[3] += a.w;
                x[4] += b.x, x[5] += b.y, x[6] += b.z, x[7] += b.w;
            }
#pragma unroll
            for (int i = 0; i < 8; ++i) x[i] = to_float(from_float<TA>(x[i]));
        } else if (!PARTS && mine) {
            const uint4 raw = *reinterpret_cast<const uint4*>((const TA*)p.proj + t * p.ld + col + d0);
            const uint32_t w[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w[i]));
                x[2 * i] = f.x, x[2 * i + 1] = f.y;
            }
        }
        if (mine) {
            if (p.bias) {
                const float4 b0 = *reinterpret_cast<const float4*>(p.bias + col + d0), b1 = *reinterpret_cast<const float4*>(p.bias + col + d0 + 4);
                x[0] += b0.x, x[1] += b0.y, x[2] += b0.z, x[3] += b0.w;
                x[4] += b1.x, x[5] += b1.y, x[6] += b1.z, x[7] += b1.w;
            }
        }
        const float* nw = is_q ? p.q_norm_w : is_v ? nullptr : p.k_norm_w;
        // every lane of the warp takes part in the sums, whichever norms its unit has
        auto norm = [&](bool wanted) {
            float ss = 0.f;
#pragma unroll
            for (int i = 0; i < 8; ++i) ss = fmaf(x[i], x[i], ss);
#pragma unroll
            for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            if (!wanted || !mine) return;
            const float r = rsqrtf(ss / (float)n + p.eps);
            if (nw) {
                const float4 a = *reinterpret_cast<const float4*>(nw + d0), b = *reinterpret_cast<const float4*>(nw + d0 + 4);
                x[0] *= r * a.x, x[1] *= r * a.y, x[2] *= r * a.z, x[3] *= r * a.w;
                x[4] *= r * b.x, x[5] *= r * b.y, x[6] *= r * b.z, x[7] *= r * b.w;
            } else {
#pragma unroll
                for (int i = 0; i < 8; ++i) x[i] *= r;
            }
        };
        if (p.qk_norm == QK_NORM_BEFORE_ROTATION || p.v_norm) norm(is_v ? p.v_norm != 0 : p.qk_norm == QK_NORM_BEFORE_ROTATION);
        if (mine && !is_v && d0 < rot) {
            const float4 cs4 = *reinterpret_cast<const float4*>(&cos_s[d0 >> 1]), sn4 = *reinterpret_cast<const float4*>(&sin_s[d0 >> 1]);
            const float cs[4] = {cs4.x, cs4.y, cs4.z, cs4.w}, sn[4] = {sn4.x, sn4.y, sn4.z, sn4.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
                if (d0 + 2 * i < rot) {
                    const float u = x[2 * i], v = x[2 * i + 1];
                    x[2 * i] = u * cs[i] - v * sn[i];
                    x[2 * i + 1] = v * cs[i] + u * sn[i];
                }
        }
        if (p.qk_norm == QK_NORM_AFTER_ROTATION) norm(!is_v);
        if (!there || d0 >= Dc) continue;
        TA* dst;
        if (is_q) {
            dst = (TA*)p.q_out + t * p.q_ld + (int64_t)head * Dc;
        } else {
            TA* cache = (TA*)(is_v ? p.v_cache : p.k_cache);
            if (!cache || !page_ok) continue;
            dst = cache + (((int64_t)page * Hkv + head) * p.page_size + pos % p.page_size) * Dc;
        }
        const float mult = (is_q && p.head_mult) ? p.head_mult[head] : 1.f;
        uint32_t o[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const __nv_bfloat162 v = __floats2bfloat162_rn(x[2 * i] * mult, x[2 * i + 1] * mult);
            o[i] = *reinterpret_cast<const uint32_t*>(&v);
        }
        *reinterpret_cast<uint4*>(dst + d0) = make_uint4(o[0], o[1], o[2], o[3]);
    }
}

// y[t, h, :] *= sigmoid(g[t, h]); a warp per (token, head).
template <typename TA>
__global__ void head_gate_kernel(TA* __restrict__ y, int64_t y_ld, const TA* __restrict__ g, int64_t g_ld, int n_tokens, int H, int Dv) {
    pdl_wait();
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31;
    const int64_t item = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (item >= (int64_t)n_tokens * H) return;
    const int64_t t = item / H;
    const int h = (int)(item - t * H);
    const float s = 1.f / (1.f + expf(-to_float(g[t * g_ld + h])));
    TA* row = y + t * y_ld + (int64_t)h * Dv;
    for (int d = lane; d < Dv; d += 32) row[d] = from_float<TA>(to_float(row[d]) * s);
}

// out[r] = ca * a[r] / rms(a[r]) * wa + cb * b[r] / rms(b[r]) * wb; one block per row, the two sums of squares in 32-bit.
template <typename TA>
__global__ void __launch_bounds__(256) rms_pair_mean_kernel(TA* __restrict__ out, const TA* __restrict__ a, const float* __restrict__ wa, float ca,
                                                            const TA* __restrict__ b, const float* __restrict__ wb, float cb, int d, float eps) {
    pdl_wait();
    pdl_launch_dependents();
    __shared__ float scratch[33];
    const int64_t r = blockIdx.x;
    const TA* ar = a + r * d;
    const TA* br = b + r * d;
    float sa = 0.f, sb = 0.f;
    for (int i = threadIdx.x; i < d; i += blockDim.x) {
        const float x = to_float(ar[i]), y = to_float(br[i]);
        sa = fmaf(x, x, sa);
        sb = fmaf(y, y, sb);
    }
    const float ra = rsqrtf(block_sum(sa, scratch) / (float)d + eps) * ca;
    const float rb = rsqrtf(block_sum(sb, scratch) / (float)d + eps) * cb;
    TA* o = out + r * d;
    for (int i = threadIdx.x; i < d; i += blockDim.x) o[i] = from_float<TA>(fmaf(to_float(ar[i]) * ra, wa[i], to_float(br[i]) * rb * wb[i]));
}

// out[t, f] = the gated activation (GateAct, kinds 0 to 2, with its bias in the rows' own order) over rows [gate | up] (block == 0) or
// runs of `block` gate entries followed by their up entries.
template <typename T>
__global__ void gated_act_kernel(T* __restrict__ out, const T* __restrict__ gu, int64_t n_tokens, int F, int block, GateAct act) {
    pdl_wait();
    pdl_launch_dependents();
    const int64_t total = n_tokens * (int64_t)F;
    for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
        const int64_t t = i / F;
        const int f = (int)(i - t * F);
        const int gi = block ? (f / block) * 2 * block + f % block : f;
        const int ui = block ? gi + block : F + f;
        const float g = to_float(gu[t * 2 * F + gi]) + (act.bias ? act.bias[gi] : 0.f);
        const float u = to_float(gu[t * 2 * F + ui]) + (act.bias ? act.bias[ui] : 0.f);
        out[i] = from_float<T>(gated_f(g, u, act));
    }
}

// out[t, j] = act(x[t, j]) for j < n: a dense copy of a slice of wider rows.  act: 0 identity, 1 tanh, 2 max(v, 0)^2.
template <typename T>
__global__ void act_rows_kernel(T* __restrict__ out, const T* __restrict__ x, int64_t ld, int64_t n_tokens, int n, int act) {
    pdl_wait();
    pdl_launch_dependents();
    const int64_t total = n_tokens * (int64_t)n;
    for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
        const int64_t t = i / n;
        const float v = to_float(x[t * ld + (i - t * n)]);
        out[i] = from_float<T>(act == 1 ? tanhf(v) : act == 2 ? relu2_f(v) : v);
    }
}


// attn [T, ld] holds, per token, G groups x 2 maps x R query heads of Dc entries (the order the paged attention kernels
// want: the R heads of a map of a group share that map's key head).  Head h = g * R + j of the result:
//   o = a[g, 0, j] - lambda * a[g, 1, j] over the first Dv entries;  y[t, h, :] = o / sqrt(mean(o^2) + eps) * out_scale.
// A warp per (token, head); the difference and the norm in 32-bit.
template <typename TA>
__global__ void diff_combine_kernel(TA* __restrict__ y, const TA* __restrict__ attn, int64_t ld, int n_tokens, int G, int R, int Dc, int Dv,
                                    const float* __restrict__ lambda, float eps, float out_scale) {
    pdl_wait();
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31;
    const int H = G * R;
    const int64_t item = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (item >= (int64_t)n_tokens * H) return;
    const int64_t t = item / H;
    const int h = (int)(item - t * H), g = h / R, j = h - g * R;
    const TA* a1 = attn + t * ld + ((int64_t)(g * 2) * R + j) * Dc;
    const TA* a2 = a1 + (int64_t)R * Dc;
    const float lam = lambda[0];
    float o[QP_MAX_D / 32], ss = 0.f;
#pragma unroll
    for (int i = 0; i < QP_MAX_D / 32; ++i) {
        const int d = lane + i * 32;
        o[i] = d < Dv ? fmaf(-lam, to_float(a2[d]), to_float(a1[d])) : 0.f;
        ss = fmaf(o[i], o[i], ss);
    }
    ss = warp_sum(ss);
    const float r = rsqrtf(ss / (float)Dv + eps) * out_scale;
    TA* dst = y + (t * H + h) * Dv;
#pragma unroll
    for (int i = 0; i < QP_MAX_D / 32; ++i) {
        const int d = lane + i * 32;
        if (d < Dv) dst[d] = from_float<TA>(o[i] * r);
    }
}

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 u;
    u.x = *reinterpret_cast<uint32_t*>(&a), u.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = u;
}

// The same with four neighbouring entries a lane (8-byte loads of 16-bit values): Dv and Dc multiples of 4, rows 8-byte aligned.
template <typename TA>
__global__ void diff_combine_vec_kernel(TA* __restrict__ y, const TA* __restrict__ attn, int64_t ld, int n_tokens, int G, int R, int Dc, int Dv,
                                        const float* __restrict__ lambda, float eps, float out_scale) {
    pdl_wait();
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31;
    const int H = G * R;
    const int64_t item = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (item >= (int64_t)n_tokens * H) return;
    const int64_t t = item / H;
    const int h = (int)(item - t * H), g = h / R, j = h - g * R;
    const TA* a1 = attn + t * ld + ((int64_t)(g * 2) * R + j) * Dc;
    const TA* a2 = a1 + (int64_t)R * Dc;
    const float lam = lambda[0];
    float4 o[QP_MAX_D / 128];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < QP_MAX_D / 128; ++i) {
        const int d = (lane + i * 32) * 4;
        o[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (d < Dv) {
            const float4 p = load4(a1 + d), q = load4(a2 + d);
            o[i] = make_float4(fmaf(-lam, q.x, p.x), fmaf(-lam, q.y, p.y), fmaf(-lam, q.z, p.z), fmaf(-lam, q.w, p.w));
        }
        ss += (o[i].x * o[i].x + o[i].y * o[i].y) + (o[i].z * o[i].z + o[i].w * o[i].w);
    }
    ss = warp_sum(ss);
    const float r = rsqrtf(ss / (float)Dv + eps) * out_scale;
    TA* dst = y + (t * H + h) * Dv;
#pragma unroll
    for (int i = 0; i < QP_MAX_D / 128; ++i) {
        const int d = (lane + i * 32) * 4;
        if (d < Dv) store4(dst + d, make_float4(o[i].x * r, o[i].y * r, o[i].z * r, o[i].w * r));
    }
}

IMP_API int imp_qkv_prepare(const ImpQkvPrepare* args, int* status, void* stream) {
    IMP_CHECK_ARG(args, "imp_qkv_prepare: null pointer");
    const ImpQkvPrepare& p = *args;
    if (p.n_tokens == 0) return 0;
    IMP_CHECK_ARG((p.proj || p.parts) && p.positions && p.seq_of_token && p.block_table && p.q_out, "imp_qkv_prepare: null pointer");
    IMP_CHECK_ARG(p.Hq > 0 && p.Hkv > 0 && p.D > 0 && p.Dv > 0 && p.Dc >= p.D && p.Dc >= p.Dv && p.Dc <= QP_MAX_D,
                  "imp_qkv_prepare: head sizes %d / %d must fit the cache's %d (at most %d)", p.D, p.Dv, p.Dc, QP_MAX_D);
    IMP_CHECK_ARG(p.rot >= 0 && p.rot % 2 == 0 && p.rot <= p.D && (p.rot == 0 || p.turns), "imp_qkv_prepare: the rotated part must be even and within the head");
    IMP_CHECK_ARG(p.qk_norm >= QK_NORM_NONE && p.qk_norm <= QK_NORM_AFTER_ROTATION && (p.q_norm_w == nullptr) == (p.k_norm_w == nullptr),
                  "imp_qkv_prepare: q and k are normalised alike");
    IMP_CHECK_ARG((p.pairing == 0 || p.pairing == 1) && p.v_share > 0 && p.Hkv % p.v_share == 0,
                  "imp_qkv_prepare: pairing is 0 (halves) or 1 (neighbours); v_share divides the key heads");
    IMP_CHECK_ARG(p.ld >= (int64_t)(p.Hq + p.Hkv) * p.D + (int64_t)(p.Hkv / p.v_share) * p.Dv && p.q_ld >= (int64_t)p.Hq * p.Dc, "imp_qkv_prepare: rows too short");
    IMP_CHECK_ARG(p.page_size > 0 && p.num_pages > 0, "imp_qkv_prepare: bad cache geometry");
    cudaStream_t s = (cudaStream_t)stream;
    const int units = p.Hq + 2 * p.Hkv;
    bool vec = p.act_dtype != IMP_F32 && p.D % 8 == 0 && p.Dv % 8 == 0 && p.Dc % 8 == 0 && p.Dc <= 256 && p.ld % 8 == 0 && p.q_ld % 8 == 0 &&
               (p.rot == 0 || p.pairing == 1);
    for (const void* q : {p.parts ? (const void*)p.parts : p.proj, (const void*)p.bias, (const void*)p.q_norm_w, (const void*)p.k_norm_w, (const void*)p.q_out, (const void*)p.k_cache,
                          (const void*)p.v_cache})
        vec = vec && (uintptr_t)q % 16 == 0;
    // few tokens: a token's units spread over several CTAs; many: one CTA makes the token's angles once for all of them
    const int per_cta = vec && p.n_tokens >= 2 * imp_sm_count() ? units : QP_UNITS;
    const dim3 grid((unsigned)p.n_tokens, (unsigned)((units + per_cta - 1) / per_cta));
    if (vec) {
#define QP_VEC(LPH)                                                                                                       \
    do {                                                                                                                  \
        if (p.parts) imp_launch(qkv_prepare_vec_kernel<LPH, true>, grid, dim3(QP_BLOCK), 0, s, p, per_cta, status);       \
        else imp_launch(qkv_prepare_vec_kernel<LPH, false>, grid, dim3(QP_BLOCK), 0, s, p, per_cta, status);              \
    } while (0)
        if (p.Dc <= 64) QP_VEC(8);
        else if (p.Dc <= 128) QP_VEC(16);
        else QP_VEC(32);
#undef QP_VEC
        IMP_RETURN_LAUNCH();
    }
#define QP_LAUNCH(TA, PER) imp_launch(qkv_prepare_kernel<TA, PER>, grid, dim3(QP_BLOCK), 0, s, p, per_cta, status)
#define QP_LAUNCH_PER(TA)                         \
    do {                                          \
        if (p.Dc <= 64) QP_LAUNCH(TA, 2);         \
        else if (p.Dc <= 128) QP_LAUNCH(TA, 4);   \
        else if (p.Dc <= 256) QP_LAUNCH(TA, 8);   \
        else QP_LAUNCH(TA, 16);                   \
    } while (0)
    if (p.act_dtype == IMP_F32) QP_LAUNCH_PER(float);
    else QP_LAUNCH_PER(__nv_bfloat16);
#undef QP_LAUNCH_PER
#undef QP_LAUNCH
    IMP_RETURN_LAUNCH();
}

// y [T, G * R * Dv] dense; attn rows `ld` apart; lambda: one float32 on the device.
IMP_API int imp_diff_combine(void* y, const void* attn, int64_t ld, int n_tokens, int G, int R, int Dc, int Dv, const float* lambda, float eps,
                             float out_scale, int dtype, void* stream) {
    if (n_tokens == 0) return 0;
    IMP_CHECK_ARG(y && attn && lambda && G > 0 && R > 0 && Dv > 0 && Dv <= Dc && Dc <= QP_MAX_D && ld >= (int64_t)2 * G * R * Dc,
                  "imp_diff_combine: bad argument");
    cudaStream_t s = (cudaStream_t)stream;
    const int64_t items = (int64_t)n_tokens * G * R;
    const dim3 grid((unsigned)((items + 7) / 8));
    const size_t el = dtype == IMP_F32 ? 4 : 2;
    if (Dv % 4 == 0 && Dc % 4 == 0 && (ld * el) % (4 * el) == 0 && (uintptr_t)attn % (4 * el) == 0 && (uintptr_t)y % (4 * el) == 0) {
        if (dtype == IMP_F32)
            imp_launch(diff_combine_vec_kernel<float>, grid, dim3(256), 0, s, (float*)y, (const float*)attn, ld, n_tokens, G, R, Dc, Dv, lambda, eps, out_scale);
        else
            imp_launch(diff_combine_vec_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, (__nv_bfloat16*)y, (const __nv_bfloat16*)attn, ld, n_tokens, G, R, Dc,
                       Dv, lambda, eps, out_scale);
        IMP_RETURN_LAUNCH();
    }
    if (dtype == IMP_F32)
        imp_launch(diff_combine_kernel<float>, grid, dim3(256), 0, s, (float*)y, (const float*)attn, ld, n_tokens, G, R, Dc, Dv, lambda, eps, out_scale);
    else
        imp_launch(diff_combine_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, (__nv_bfloat16*)y, (const __nv_bfloat16*)attn, ld, n_tokens, G, R, Dc, Dv,
                   lambda, eps, out_scale);
    IMP_RETURN_LAUNCH();
}

IMP_API int imp_head_gate(void* y, int64_t y_ld, const void* g, int64_t g_ld, int n_tokens, int H, int Dv, int dtype, void* stream) {
    if (n_tokens == 0) return 0;
    IMP_CHECK_ARG(y && g && H > 0 && Dv > 0 && y_ld >= (int64_t)H * Dv && g_ld >= H, "imp_head_gate: bad argument");
    cudaStream_t s = (cudaStream_t)stream;
    const int64_t items = (int64_t)n_tokens * H;
    const dim3 grid((unsigned)((items + 7) / 8));
    if (dtype == IMP_F32) imp_launch(head_gate_kernel<float>, grid, dim3(256), 0, s, (float*)y, y_ld, (const float*)g, g_ld, n_tokens, H, Dv);
    else imp_launch(head_gate_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, (__nv_bfloat16*)y, y_ld, (const __nv_bfloat16*)g, g_ld, n_tokens, H, Dv);
    IMP_RETURN_LAUNCH();
}

IMP_API int imp_rms_pair_mean(void* out, const void* a, const float* wa, float ca, const void* b, const float* wb, float cb, int n_rows, int d,
                              float eps, int dtype, void* stream) {
    if (n_rows == 0) return 0;
    IMP_CHECK_ARG(out && a && b && wa && wb && d > 0, "imp_rms_pair_mean: bad argument");
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == IMP_F32)
        imp_launch(rms_pair_mean_kernel<float>, dim3(n_rows), dim3(256), 0, s, (float*)out, (const float*)a, wa, ca, (const float*)b, wb, cb, d, eps);
    else
        imp_launch(rms_pair_mean_kernel<__nv_bfloat16>, dim3(n_rows), dim3(256), 0, s, (__nv_bfloat16*)out, (const __nv_bfloat16*)a, wa, ca,
                   (const __nv_bfloat16*)b, wb, cb, d, eps);
    IMP_RETURN_LAUNCH();
}

IMP_API int imp_gated_act(void* out, const void* gate_up, int n_tokens, int F, int block, int act, float limit, const float* bias, int dtype,
                          void* stream) {
    if (n_tokens == 0 || F == 0) return 0;
    IMP_CHECK_ARG(out && gate_up && n_tokens > 0 && F > 0 && block >= 0 && (block == 0 || F % block == 0) && act >= ACT_SILU && act <= ACT_CLIPPED,
                  "imp_gated_act: bad argument");
    cudaStream_t s = (cudaStream_t)stream;
    const int64_t total = (int64_t)n_tokens * F;
    const dim3 grid((unsigned)std::min<int64_t>((total + 255) / 256, 65535));
    if (dtype == IMP_F32) imp_launch(gated_act_kernel<float>, grid, dim3(256), 0, s, (float*)out, (const float*)gate_up, (int64_t)n_tokens, F, block, GateAct(act, limit, bias));
    else imp_launch(gated_act_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, (__nv_bfloat16*)out, (const __nv_bfloat16*)gate_up, (int64_t)n_tokens, F, block, GateAct(act, limit, bias));
    IMP_RETURN_LAUNCH();
}

IMP_API int imp_act_rows(void* out, const void* x, int64_t ld, int n_tokens, int n, int act, int dtype, void* stream) {
    if (n_tokens == 0 || n == 0) return 0;
    IMP_CHECK_ARG(out && x && n > 0 && ld >= n && act >= 0 && act <= 2, "imp_act_rows: bad argument");
    cudaStream_t s = (cudaStream_t)stream;
    const int64_t total = (int64_t)n_tokens * n;
    const dim3 grid((unsigned)std::min<int64_t>((total + 255) / 256, 65535));
    if (dtype == IMP_F32) imp_launch(act_rows_kernel<float>, grid, dim3(256), 0, s, (float*)out, (const float*)x, ld, (int64_t)n_tokens, n, act);
    else imp_launch(act_rows_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, (__nv_bfloat16*)out, (const __nv_bfloat16*)x, ld, (int64_t)n_tokens, n, act);
    IMP_RETURN_LAUNCH();
}

// dst[t, h, 0:n] = src[t, h, 0:n] out of heads of `ds` entries: the heads' first n columns as dense rows.
template <typename T>
__global__ void gather_head_cols_kernel(T* __restrict__ dst, const T* __restrict__ src, int64_t n_tokens, int H, int ds, int n) {
    pdl_wait();
    pdl_launch_dependents();
    const int64_t total = n_tokens * (int64_t)H * n;
    for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
        const int64_t th = i / n;
        dst[i] = src[th * ds + (i - th * n)];
    }
}

IMP_API int imp_gather_head_cols(void* dst, const void* src, int n_tokens, int H, int ds, int n, int dtype, void* stream) {
    if (n_tokens == 0) return 0;
    IMP_CHECK_ARG(dst && src && H > 0 && n > 0 && ds >= n, "imp_gather_head_cols: bad argument");
    cudaStream_t s = (cudaStream_t)stream;
    const int64_t total = (int64_t)n_tokens * H * n;
    const dim3 grid((unsigned)std::min<int64_t>((total + 255) / 256, 65535));
    if (dtype == IMP_F32) imp_launch(gather_head_cols_kernel<float>, grid, dim3(256), 0, s, (float*)dst, (const float*)src, (int64_t)n_tokens, H, ds, n);
    else imp_launch(gather_head_cols_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, (__nv_bfloat16*)dst, (const __nv_bfloat16*)src, (int64_t)n_tokens, H, ds, n);
    IMP_RETURN_LAUNCH();
}
