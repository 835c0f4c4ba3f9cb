// Arguments of imp_qkv_prepare (qkv_prepare.cu): what stands between a q,k,v product and the paged attention kernels.
#pragma once

#include <stdint.h>

enum { QK_NORM_NONE = 0, QK_NORM_BEFORE_ROTATION = 1, QK_NORM_AFTER_ROTATION = 2 };

struct ImpQkvPrepare {
    const void* proj = nullptr;        // [n_tokens, ld] in act_dtype, columns [q: Hq * D | k: Hkv * D | v: (Hkv / v_share) * Dv | ...]
    int64_t ld = 0;
    const float* parts = nullptr;      // instead of proj: the unsummed float32 parts [n_splits][n_tokens, ld] of the product, added
    int n_splits = 0;                  // in order and rounded to act_dtype as the summing kernel would have stored them
    const float* bias = nullptr;       // one number per column of q, k and v, added first; or null
    int n_tokens = 0, Hq = 0, Hkv = 0, D = 0, Dv = 0;
    int Dc = 0;                        // the cache's head size (at least D and Dv): the rest of a row is zeros
    int qk_norm = QK_NORM_NONE;        // an RMS norm over the D entries of every q and k head
    const float* q_norm_w = nullptr;   // its weights [D], shared by the heads; null: none
    const float* k_norm_w = nullptr;
    float eps = 0.f;                   // of the norms of q, k and v
    int v_norm = 0;                    // values divided by their root mean square
    const float* turns = nullptr;      // [2][rot / 2]: a pair's turns (angle / 2 pi) per position, as the sum of two floats
    int rot = 0;                       // entries of a head that are rotated (even; 0: none)
    int pairing = 0;                   // 0: entry i with i + rot / 2; 1: neighbours 2i, 2i + 1
    float rot_mult = 1.f;              // a factor on cos and sin
    int v_share = 1;                   // neighbouring key heads that cache copies of one value head
    const float* head_mult = nullptr;  // a factor per query head, or null
    const int* positions = nullptr;
    const int* seq_of_token = nullptr;
    const int* block_table = nullptr;
    int bt_stride = 0, n_seqs = 0;
    void* q_out = nullptr;             // [n_tokens, q_ld], heads of Dc entries
    int64_t q_ld = 0;
    void* k_cache = nullptr;           // pages [page][kv head][slot][Dc]; null: nothing is written
    void* v_cache = nullptr;
    int page_size = 0, num_pages = 0, act_dtype = 0;
};
