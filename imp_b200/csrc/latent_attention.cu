// The small kernels of latent attention: what happens between its matrix products.
//
// A token's down-projection holds [ query latent (q_rank) | key/value latent (kv_rank) | rotated key part (rot) ].
// (a model without a query latent has q_rank 0).  latent_prepare: RMS norm (plain weight, eps inside the root) of the two latents, rotation of the key part at the
// token's position, and the cache write: a page holds one vector [kv_rank + rot] per token, the normalised latent
// followed by the rotated key part.  latent_query_rope: the rotated part of every head's query, moved behind that
// head's latent-space query; latent_prepare can do this as well, where the query's product is done before it.  A page's vector
// and a head's query may be padded with zeros to a whole multiple of 16.  Norms, angles and rotations are 32-bit; the rotation
// pairs entry i with i + dims/2 (pairing 0) or 2i with 2i + 1 (pairing 1).
#include <algorithm>

#include "common.cuh"

namespace {

constexpr int LP_BLOCK = 128, LP_BLOCK_MAX = 256;

// Entry i of a rotated vector `x` (its first rot_dims entries turn, the rest stays); cos/sin: the position's row of the tables.
template <typename TA>
__device__ __forceinline__ float rotated_entry(const TA* __restrict__ x, int i, int rot_dims, int pairing, const float* __restrict__ cos_row,
                                               const float* __restrict__ sin_row) {
    const float v = to_float(x[i]);
    if (i >= rot_dims) return v;
    const int half = rot_dims / 2;
    const int f = pairing ? i >> 1 : (i < half ? i : i - half);
    const bool first = pairing ? (i & 1) == 0 : i < half;
    const float other = to_float(x[pairing ? i ^ 1 : (first ? i + half : i - half)]);
    return first ? v * cos_row[f] - other * sin_row[f] : v * cos_row[f] + other * sin_row[f];
}

// The rotated parts of a token's query heads, for a prepare kernel that makes them too: head h's part starts at
// q + h * q_head and goes to out + h * out_head, followed by `pad` zeros.  H == 0: nothing to do.
template <typename TA> struct QueryParts {
    const TA* q;
    int64_t q_ld;
    int q_head;
    TA* out;
    int64_t out_ld;
    int out_head, H, pad;
};

template <typename TA>
__global__ void __launch_bounds__(LP_BLOCK_MAX) latent_prepare_kernel(
    const TA* __restrict__ proj, int64_t ld, int q_rank, int kv_rank, int rot, const float* __restrict__ wq, const float* __restrict__ wkv,
    float eps, TA* __restrict__ cq, int64_t cq_ld, const float* __restrict__ cos_tab, const float* __restrict__ sin_tab, int rot_dims,
    int pairing, int max_pos, const int* __restrict__ positions, const int* __restrict__ seq_of_token, const int* __restrict__ block_table,
    int bt_stride, int n_seqs, TA* __restrict__ pages, int page_len, int page_size, int num_pages, QueryParts<TA> qp, int* status) {
    pdl_wait();
    pdl_launch_dependents();
    __shared__ float scratch[33];
    const int t = blockIdx.x, tid = threadIdx.x, n_thr = blockDim.x;
    const TA* row = proj + (int64_t)t * ld;
    float ss = 0.f, inv;
    // CTA (t, 0) does the norms and the cache write of token t, CTAs (t, 1 ...) share its query heads
    const bool query_cta = blockIdx.y > 0;
    if (q_rank > 0 && !query_cta) {
        // the query latent
        for (int i = tid; i < q_rank; i += n_thr) {
            const float v = to_float(row[i]);
            ss = fmaf(v, v, ss);
        }
        inv = rsqrtf(block_sum(ss, scratch) / (float)q_rank + eps);
        for (int i = tid; i < q_rank; i += n_thr) cq[(int64_t)t * cq_ld + i] = from_float<TA>(to_float(row[i]) * inv * wq[i]);
    }
    const int seq = seq_of_token[t], pos = positions[t];
    if (!pages && qp.H == 0) return;
    if (seq < 0 || seq >= n_seqs || pos < 0 || pos >= max_pos || (pages && pos / page_size >= bt_stride)) {
        if (tid == 0) imp_report(status, seq < 0 || seq >= n_seqs ? IMP_BAD_SEQUENCE : IMP_BAD_POSITION);
        return;
    }
    const float* cos_row = cos_tab + (int64_t)pos * (rot_dims / 2);
    const float* sin_row = sin_tab + (int64_t)pos * (rot_dims / 2);
    if (query_cta) {
        // the rotated part of every head's query, behind that head's latent-space query
        const int per = rot + qp.pad;
        for (int e = (blockIdx.y - 1) * n_thr + tid; e < qp.H * per; e += (gridDim.y - 1) * n_thr) {
            const int h = e / per, i = e - h * per;
            const TA* src = qp.q + (int64_t)t * qp.q_ld + (int64_t)h * qp.q_head;
            qp.out[(int64_t)t * qp.out_ld + (int64_t)h * qp.out_head + i] =
                from_float<TA>(i < rot ? rotated_entry(src, i, rot_dims, pairing, cos_row, sin_row) : 0.f);
        }
        return;
    }
    // the key/value latent and the rotated key part go to the token's place in the pages
    if (!pages) return;
    const int page = block_table[(int64_t)seq * bt_stride + pos / page_size];
    if (page < 0 || page >= num_pages) {
        if (tid == 0) imp_report(status, IMP_BAD_PAGE);
        return;
    }
    TA* dst = pages + ((int64_t)page * page_size + pos % page_size) * page_len;
    const TA* lat = row + q_rank;
    ss = 0.f;
    for (int i = tid; i < kv_rank; i += n_thr) {
        const float v = to_float(lat[i]);
        ss = fmaf(v, v, ss);
    }
    inv = rsqrtf(block_sum(ss, scratch) / (float)kv_rank + eps);
    for (int i = tid; i < kv_rank; i += n_thr) dst[i] = from_float<TA>(to_float(lat[i]) * inv * wkv[i]);
    const TA* kr = lat + kv_rank;
    for (int i = tid; i < page_len - kv_rank; i += n_thr)
        dst[kv_rank + i] = from_float<TA>(i < rot ? rotated_entry(kr, i, rot_dims, pairing, cos_row, sin_row) : 0.f);
}

// q [T, H, D + rot] -> out[t, h, kv_rank + i] = rotated q[t, h, D + i]
template <typename TA>
__global__ void latent_query_rope_kernel(const TA* __restrict__ q, int64_t q_ld, int H, int D, int rot, TA* __restrict__ out, int64_t out_ld,
                                         int kv_rank, const float* __restrict__ cos_tab, const float* __restrict__ sin_tab, int rot_dims,
                                         int max_pos, const int* __restrict__ positions, int* status) {
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x;
    const int pos = positions[t];
    if (pos < 0 || pos >= max_pos) {
        if (threadIdx.x == 0) imp_report(status, IMP_BAD_POSITION);
        return;
    }
    const int half = rot_dims / 2;
    for (int e = threadIdx.x; e < H * rot; e += blockDim.x) {
        const int h = e / rot, i = e % rot;
        const TA* src = q + (int64_t)t * q_ld + (int64_t)h * (D + rot) + D;
        const float v = rotated_entry(src, i, rot_dims, 0, cos_tab + (int64_t)pos * half, sin_tab + (int64_t)pos * half);
        out[(int64_t)t * out_ld + (int64_t)h * (kv_rank + rot) + kv_rank + i] = from_float<TA>(v);
    }
}

}  // namespace

namespace {
template <typename TA>
cudaError_t launch_prepare(const void* proj, int64_t ld, int n_tokens, int q_rank, int kv_rank, int rot, const float* wq, const float* wkv, float eps,
                           void* cq, int64_t cq_ld, const float* cos_tab, const float* sin_tab, int rot_dims, int pairing, int max_pos,
                           const int* positions, const int* seq_of_token, const int* block_table, int bt_stride, int n_seqs, void* pages,
                           int page_len, int page_size, int num_pages, const void* q, int64_t q_ld, int q_head, void* q_out, int64_t q_out_ld, int H,
                           int* status, cudaStream_t s) {
    QueryParts<TA> qp{(const TA*)q, q_ld, q_head, (TA*)q_out, q_out_ld, page_len, q ? H : 0, page_len - kv_rank - rot};
    // a step of few tokens spreads a token's query heads over several CTAs
    const int block = qp.H * rot > 512 ? LP_BLOCK_MAX : LP_BLOCK, work = (qp.H * (page_len - kv_rank) + block - 1) / block;
    const int query_ctas = qp.H > 0 ? std::max(1, std::min(work, 2 * imp_sm_count() / std::max(n_tokens, 1))) : 0;
    return imp_launch(latent_prepare_kernel<TA>, dim3(n_tokens, 1 + query_ctas), dim3(block), 0, s, (const TA*)proj, ld, q_rank,
                      kv_rank, rot, wq, wkv, eps, (TA*)cq, cq_ld, cos_tab, sin_tab, rot_dims, pairing, max_pos, positions, seq_of_token, block_table,
                      bt_stride, n_seqs, (TA*)pages, page_len, page_size, num_pages, qp, status);
}
}  // namespace

// proj rows: [query latent (q_rank, may be 0) | key/value latent | rotated key part].  page_len >= kv_rank + rot: the length of a
// page's vector, zeros behind the rotated part.  pairing: 0 halves, 1 neighbours.  q (may be null): the rotated part of head 0's
// query of token 0, heads q_head entries apart; it goes, rotated, to q_out + h * page_len, zeros behind it.
IMP_API int imp_latent_prepare_ex(const void* proj, int64_t ld, int n_tokens, int q_rank, int kv_rank, int rot, const float* wq, const float* wkv,
                                  float eps, void* cq, int64_t cq_ld, const float* cos_tab, const float* sin_tab, int rot_dims, int pairing,
                                  int max_pos, const int* positions, const int* seq_of_token, const int* block_table, int bt_stride, int n_seqs,
                                  void* pages, int page_len, int page_size, int num_pages, const void* q, int64_t q_ld, int q_head, void* q_out,
                                  int64_t q_out_ld, int H, int act_dtype, int* status, void* stream) {
    if (n_tokens == 0) return 0;
    IMP_CHECK_ARG(proj && (q_rank == 0 || (wq && cq)) && wkv && cos_tab && sin_tab && positions && seq_of_token, "imp_latent_prepare: null pointer");
    IMP_CHECK_ARG(q_rank >= 0 && kv_rank > 0 && rot >= 0 && rot_dims >= 0 && rot_dims <= rot && rot_dims % 2 == 0 && page_len >= kv_rank + rot,
                  "imp_latent_prepare: bad sizes (the rotated entries must be even in number and within the rotated part)");
    IMP_CHECK_ARG(!pages || (block_table && page_size > 0 && num_pages > 0), "imp_latent_prepare: bad cache geometry");
    IMP_CHECK_ARG((pairing == 0 || pairing == 1) && (!q || (q_out && H > 0 && q_head >= rot)), "imp_latent_prepare: bad query parts or pairing");
    cudaStream_t s = (cudaStream_t)stream;
    cudaError_t e;
    if (act_dtype == IMP_F32)
        e = launch_prepare<float>(proj, ld, n_tokens, q_rank, kv_rank, rot, wq, wkv, eps, cq, cq_ld, cos_tab, sin_tab, rot_dims, pairing, max_pos,
                                  positions, seq_of_token, block_table, bt_stride, n_seqs, pages, page_len, page_size, num_pages, q, q_ld, q_head, q_out,
                                  q_out_ld, H, status, s);
    else
        e = launch_prepare<__nv_bfloat16>(proj, ld, n_tokens, q_rank, kv_rank, rot, wq, wkv, eps, cq, cq_ld, cos_tab, sin_tab, rot_dims, pairing,
                                          max_pos, positions, seq_of_token, block_table, bt_stride, n_seqs, pages, page_len, page_size, num_pages, q,
                                          q_ld, q_head, q_out, q_out_ld, H, status, s);
    if (e != cudaSuccess) {
        imp_set_error("imp_latent_prepare: %s", cudaGetErrorString(e));
        return (int)e;
    }
    return 0;
}

IMP_API int imp_latent_prepare(const void* proj, int64_t ld, int n_tokens, int q_rank, int kv_rank, int rot, const float* wq,
                               const float* wkv, float eps, void* cq, int64_t cq_ld, const float* cos_tab, const float* sin_tab,
                               int rot_dims, int max_pos, const int* positions, const int* seq_of_token, const int* block_table,
                               int bt_stride, int n_seqs, void* pages, int page_size, int num_pages, int act_dtype, int* status,
                               void* stream) {
    return imp_latent_prepare_ex(proj, ld, n_tokens, q_rank, kv_rank, rot, wq, wkv, eps, cq, cq_ld, cos_tab, sin_tab, rot_dims, 0, max_pos, positions,
                                 seq_of_token, block_table, bt_stride, n_seqs, pages, kv_rank + rot, page_size, num_pages, nullptr, 0, 0, nullptr, 0, 0,
                                 act_dtype, status, stream);
}

IMP_API int imp_latent_query_rope(const void* q, int64_t q_ld, int n_tokens, int H, int D, int rot, void* out, int64_t out_ld, int kv_rank,
                                  const float* cos_tab, const float* sin_tab, int rot_dims, int max_pos, const int* positions,
                                  int act_dtype, int* status, void* stream) {
    if (n_tokens == 0 || rot == 0) return 0;
    IMP_CHECK_ARG(q && out && cos_tab && sin_tab && positions && H > 0 && D >= 0 && rot > 0 && rot_dims <= rot && rot_dims % 2 == 0,
                  "imp_latent_query_rope: bad argument");
    cudaStream_t s = (cudaStream_t)stream;
    cudaError_t e;
    if (act_dtype == IMP_F32)
        e = imp_launch(latent_query_rope_kernel<float>, dim3(n_tokens), dim3(128), 0, s, (const float*)q, q_ld, H, D, rot, (float*)out, out_ld,
                       kv_rank, cos_tab, sin_tab, rot_dims, max_pos, positions, status);
    else
        e = imp_launch(latent_query_rope_kernel<__nv_bfloat16>, dim3(n_tokens), dim3(128), 0, s, (const __nv_bfloat16*)q, q_ld, H, D, rot,
                       (__nv_bfloat16*)out, out_ld, kv_rank, cos_tab, sin_tab, rot_dims, max_pos, positions, status);
    if (e != cudaSuccess) {
        imp_set_error("imp_latent_query_rope: %s", cudaGetErrorString(e));
        return (int)e;
    }
    return 0;
}
