// Part kinds: layer norm, latent attention, the wkv recurrence, routed experts with a shared expert, a pre-norm block
// whose branches carry a learned factor per channel, and a block that re-makes the stream from itself and the
// embedding's output.  Every size and constant is a parameter; no kind knows which model it is in.
#include <cmath>

#include "kernels.h"
#include "ops.hpp"
#include "parts.hpp"

namespace imp {

namespace {

int64_t need_int(const Json& p, const char* key, const char* part) {
    const Json* v = p.find(key);
    if (!v || !v->is_number()) fail(IMP_ERROR_INVALID_MODEL, std::string(part) + ": parameter '" + key + "' is missing");
    return v->as_int();
}
double need_double(const Json& p, const char* key, const char* part) {
    const Json* v = p.find(key);
    if (!v || !v->is_number()) fail(IMP_ERROR_INVALID_MODEL, std::string(part) + ": parameter '" + key + "' is missing");
    return v->as_double();
}

// A branch whose unsummed parts, if any, have been added up; a factor per column stays with it.
Branch parts_summed(Runtime& rt, const Branch& b) {
    if (!b.split()) return b;
    Branch plain = b;
    plain.col_scale = nullptr;
    plain.own_norm = BranchNorm{};
    Branch out = Branch::of(summed(rt, plain));
    out.col_scale = b.col_scale;
    out.own_norm = b.own_norm;
    return out;
}

// -------------------------------------------------------------------------------------------- layer norm
// y = (x - mean) / sqrt(var + eps) * w (+ b) over the last axis, the variance being the mean of the squared deviations; a
// weight and, with `bias`, a bias.  Statistics in 32-bit.  It can store its result as the stream (post-norm blocks).
// params: size, eps, bias (default false).
struct LayerNorm : Norm {
    Tensor weight, bias{};
    float eps;
    explicit LayerNorm(BuildArgs& a) : weight(a.tensor("weight")), eps((float)a.params.get_double("eps", 1e-5)) {
        if (a.params.get_bool("bias", false)) {
            bias = a.tensor("bias");
            if (bias.dtype != weight.dtype || numel(bias) != numel(weight)) fail(IMP_ERROR_INVALID_MODEL, "layernorm: weight and bias must agree in type and size");
        }
    }
    bool takes_column_scale() const override { return true; }
    bool takes_normed_branch() const override { return true; }
    bool as_branch_norm(BranchNorm* out) const override {
        out->weight = weight.data;
        out->bias = bias.data;
        out->eps = eps;
        out->dtype = weight.dtype;
        return true;
    }
    bool stores_stream() const override { return true; }
    // A branch with a norm of its own that this kernel family cannot apply while adding (another weight type, or factors per
    // column as well) gets it applied first.
    Branch plain_or_normed(Runtime& rt, const Branch& branch) const {
        Branch b = parts_summed(rt, branch);
        if (b.own_norm.weight && (b.col_scale || b.own_norm.dtype != weight.dtype)) b = Branch::of(summed(rt, b));
        return b;
    }
    Tensor add_norm_store(Step& st, Tensor h, float h_mult, const Branch& branch) override {
        Runtime& rt = *st.rt;
        const int d = (int)cols(h);
        Tensor out = rt.empty(rows(h), d);
        if (h.dtype != F32 || !contiguous(h) || numel(weight) != d) fail(IMP_ERROR_INVALID_ARG, "layernorm: the stream must be dense float32 [T, d], the weight [d]");
        Branch b = parts_summed(rt, branch);
        if (b.own_norm.weight) b = Branch::of(summed(rt, b));
        if (!b.empty() && (rows(b.t) != rows(h) || cols(b.t) != d || b.t.dtype != out.dtype || !contiguous(b.t)))
            fail(IMP_ERROR_INVALID_ARG, "layernorm: the branch must be dense, of the stream's shape and the output's type");
        ++rt.launches;
        check_launch(imp_add_layernorm_ex((float*)h.data, h_mult, b.empty() ? nullptr : b.t.data, b.col_scale, weight.data, bias.data, out.data, nullptr,
                                          (int)rows(h), d, eps, out.dtype, weight.dtype, 2, rt.stream),
                     "add_layernorm");
        return out;
    }
    Tensor add_norm(Step& st, Tensor h, const Branch& branch, const int32_t* rows_idx, int n_rows) override {
        Runtime& rt = *st.rt;
        const int64_t n = rows_idx ? n_rows : rows(h);
        const int d = (int)cols(h);
        Tensor out = rt.empty(n, d, -1, /*step=*/rows_idx != nullptr);
        if (h.dtype != F32 || !contiguous(h) || numel(weight) != d) fail(IMP_ERROR_INVALID_ARG, "layernorm: the stream must be dense float32 [T, d], the weight [d]");
        const Branch b = plain_or_normed(rt, branch);
        if (!b.empty() && (rows(b.t) != rows(h) || cols(b.t) != d || b.t.dtype != out.dtype || !contiguous(b.t)))
            fail(IMP_ERROR_INVALID_ARG, "layernorm: the branch must be dense, of the stream's shape and the output's type");
        ++rt.launches;
        if (b.own_norm.weight && st.row_op && !rows_idx) {
            // ... and the per-row operation of the rows' reader behind it, where the kernel's form takes it
            RowOp& op = *st.row_op;
            const int rc = imp_add_normed_layernorm_conv((float*)h.data, b.t.data, b.own_norm.weight, b.own_norm.bias, b.own_norm.eps, weight.data, bias.data,
                                                         eps, out.data, (int)n, d, out.dtype, weight.dtype, op.conv_w, op.taps, op.conv_state,
                                                         st.view.seq_of_token, st.view.state_slots, rt.stream);
            if (rc == 0) {
                op.taken = true;
                return out;
            }
            if (rc != -2) check_launch(rc, "add_normed_layernorm_conv");   // -2: the kernel declined (width or alignment); the unfused launches follow
        }
        if (b.own_norm.weight) {
            // the branch's own norm, the sum and this norm in one pass
            check_launch(imp_add_normed_layernorm((float*)h.data, b.t.data, b.own_norm.weight, b.own_norm.bias, b.own_norm.eps, weight.data, bias.data, eps,
                                                  out.data, rows_idx, (int)n, d, out.dtype, weight.dtype, rows_idx ? 0 : 1, rt.stream),
                         "add_normed_layernorm");
            return out;
        }
        check_launch(imp_add_layernorm_ex((float*)h.data, 1.f, b.empty() ? nullptr : b.t.data, b.col_scale, weight.data, bias.data, out.data, rows_idx,
                                          (int)n, d, eps, out.dtype, weight.dtype, rows_idx ? 0 : 1, rt.stream),
                     "add_layernorm");
        return out;
    }
};

// ------------------------------------------------------------------------------------- latent attention
// Causal softmax attention whose keys and values are expanded from a small latent per token:
//   c_q = rms(W_dq x) * n_q;  q = W_uq c_q, per head [D plain | R rotated]
//   W_dkv x = [ latent (C) | rotated key part (R) ];  c = rms(latent) * n_kv;  the key part is one for all heads
//   per head: k_plain = W_uk c, v = W_uv c;  score = scale * (q_plain . k_plain + rot(q_rot) . rot(k_rot))
//   out = W_o [heads' softmax-weighted values]
// Only c and the rotated key part are cached: one vector [C + R] per token, keys only.  The products with W_uk and W_uv
// are moved to the query side and the output side: q_lat = W_uk^T q_plain lives in the latent space, attention runs as
// one shared "kv head" of size C + R over the cache (the pages serve as keys and as values; the last R entries of its
// output are not used), and W_uv maps each head's latent-space result to its values.  Per token the cache holds
// C + R numbers whatever the number of heads.
//
// Options: no query latent (`q_rank` 0: q = W_q x, a tensor `q_proj`); a sliding window (`window`: the last so many keys, 0 all);
// the rotation's pairing (`rot_pairing`: "halves" i, i + rot_dims/2 | "neighbours" 2i, 2i + 1); the heads' values multiplied by
// sigmoid(W_g x) before W_o (`out_gate`: a tensor `gate_proj`); the cached vector padded with zeros to a multiple of 16 where the
// tensor-core kernels then take it (`pad_cache`).  Without a query latent all of x's projections are one product.
//
// params: hidden_size, num_heads, head_dim (plain), rot_dim, value_dim, kv_rank, q_rank, scale, norm_eps, rot_base,
//         rot_dims (entries of the rotated part that are rotated: even, at most rot_dim), max_positions, window, rot_pairing,
//         out_gate, pad_cache.
struct LatentAttention : Mixer {
    int H, D, R, Dv, C, Q, L, rot_dims, pairing = 0;   // L: the length of a cached vector
    bool gated = false;
    float eps;
    AttentionGeometry g;
    int64_t gate_col = 0;
    Tensor w_down, w_uq, w_ukT, w_uv, w_o, n_q, n_kv;
    Position* position = nullptr;

    struct Sizes {
        int64_t d, H, D, R, Dv, C, Q, L;
    };
    static Sizes sizes(const Json& p) {
        const char* me = "latent_attention";
        Sizes s{need_int(p, "hidden_size", me), need_int(p, "num_heads", me), need_int(p, "head_dim", me), need_int(p, "rot_dim", me),
                need_int(p, "value_dim", me), need_int(p, "kv_rank", me), need_int(p, "q_rank", me), 0};
        s.L = s.C + s.R;
        if (p.get_bool("pad_cache", false) && s.L <= 256) s.L = (s.L + 15) / 16 * 16;
        if (s.H <= 0 || s.D <= 0 || s.R <= 0 || s.Dv <= 0 || s.C <= 0 || s.Q < 0) fail(IMP_ERROR_INVALID_MODEL, std::string(me) + ": every size must be positive");
        if (s.Q > 0 && (s.L != s.C + s.R || p.get_string("rot_pairing", "halves") != "halves"))
            fail(IMP_ERROR_UNSUPPORTED, std::string(me) + ": a query latent goes with rotated halves and an unpadded cache");
        if (s.C + s.R > 1024)
            fail(IMP_ERROR_INVALID_MODEL, std::string(me) + ": kv_rank + rot_dim = " + std::to_string(s.C + s.R) + " exceeds the attention kernels' 1024 (tensor cores up to 256)");
        return s;
    }
    static TensorSpecs specs(const Json& p) {
        const Sizes z = sizes(p);
        TensorSpecs s;
        if (z.Q > 0) {
            s.emplace_back("q_down", TensorSpec{{z.Q, z.d}});
            s.emplace_back("q_norm", TensorSpec{{z.Q}, "norm", "one_plus_normal"});
            s.emplace_back("q_up", TensorSpec{{z.H * (z.D + z.R), z.Q}});
        } else {
            s.emplace_back("q_proj", TensorSpec{{z.H * (z.D + z.R), z.d}});
        }
        s.emplace_back("kv_down", TensorSpec{{z.C + z.R, z.d}});
        s.emplace_back("kv_norm", TensorSpec{{z.C}, "norm", "one_plus_normal"});
        s.emplace_back("k_up", TensorSpec{{z.H * z.D, z.C}});
        s.emplace_back("v_up", TensorSpec{{z.H * z.Dv, z.C}});
        if (p.get_bool("out_gate", false)) s.emplace_back("gate_proj", TensorSpec{{z.H * z.Dv, z.d}});
        s.emplace_back("o_proj", TensorSpec{{z.d, z.H * z.Dv}});
        return s;
    }
    static CacheSpec cache(const Json& p) {
        const Sizes z = sizes(p);
        CacheSpec s = CacheSpec::paged(1, (int)z.L, (int)p.get_int("window", 0));
        s.keys_only = true;
        return s;
    }

    explicit LatentAttention(BuildArgs& a) {
        const char* me = "latent_attention";
        const Sizes z = sizes(a.params);
        H = (int)z.H, D = (int)z.D, R = (int)z.R, Dv = (int)z.Dv, C = (int)z.C, Q = (int)z.Q, L = (int)z.L;
        gated = a.params.get_bool("out_gate", false);
        const std::string pr = a.params.get_string("rot_pairing", "halves");
        if (pr != "neighbours" && pr != "halves") fail(IMP_ERROR_INVALID_MODEL, std::string(me) + ": unknown rot_pairing '" + pr + "' (known: neighbours, halves)");
        pairing = pr == "neighbours" ? 1 : 0;
        rot_dims = (int)a.params.get_int("rot_dims", R);
        if (rot_dims < 2 || rot_dims % 2 || rot_dims > R)
            fail(IMP_ERROR_INVALID_MODEL, std::string(me) + ": rot_dims " + std::to_string(rot_dims) + " must be even and within rot_dim " + std::to_string(R));
        eps = (float)a.params.get_double("norm_eps", 1e-6);
        g.hq = H, g.hkv = 1, g.dh = L, g.window = (int)a.params.get_int("window", 0);
        if (g.window < 0) fail(IMP_ERROR_INVALID_MODEL, std::string(me) + ": 'window' must not be negative");
        g.scale = (float)need_double(a.params, "scale", me);
        Runtime& rt = *a.rt;
        // one product for everything that reads x: [query latent or q | latent and rotated key part | gate], the gate starting on a
        // multiple of 8 columns and the rows padded to one
        std::vector<Tensor> in = {a.tensor(Q > 0 ? "q_down" : "q_proj"), a.tensor("kv_down")}, pads;
        int64_t n = (Q > 0 ? z.Q : z.H * (z.D + z.R)) + z.C + z.R;
        auto pad_to8 = [&] {
            const int64_t pad = (8 - n % 8) % 8;
            if (!pad) return;
            Tensor zeros = a.store->alloc(in[0].dtype, {pad, z.d});
            IMP_CUDA(cudaMemsetAsync(zeros.data, 0, (size_t)numel(zeros) * elem_size(zeros.dtype), rt.stream));
            in.push_back(zeros);
            pads.push_back(zeros);
            n += pad;
        };
        pad_to8();
        if (gated) {
            gate_col = n;
            in.push_back(a.tensor("gate_proj"));
            n += z.H * z.Dv;
            pad_to8();
        }
        w_down = cat_rows(rt, *a.store, in);
        if (Q > 0) w_uq = a.tensor("q_up");
        w_uv = a.tensor("v_up");
        w_o = a.tensor("o_proj");
        // W_uk [H][D, C] -> [H][C, D]: the latent-space query is a product with W_uk's transpose
        const Tensor uk = a.tensor("k_up");
        w_ukT = a.store->alloc(uk.dtype, {z.H * z.C, z.D});
        check_launch(imp_transpose_groups(w_ukT.data, uk.data, H, D, C, uk.dtype == F32 ? 0 : 1, rt.stream), "transpose_groups");
        if (Q > 0) n_q = to_float32(rt, *a.store, a.tensor("q_norm"));
        n_kv = to_float32(rt, *a.store, a.tensor("kv_norm"));
        Json pos = Json::object(), pp = Json::object();
        pos["kind"] = "rotary";
        pp["head_dim"] = (int64_t)R;
        pp["rotary_dim"] = (int64_t)rot_dims;
        pp["theta"] = need_double(a.params, "rot_base", me);
        pp["max_positions"] = need_int(a.params, "max_positions", me);
        pos["params"] = pp;
        position = part_cast<Position>(a.factory->shared("position", pos), "a position encoding");
        IMP_CUDA(cudaStreamSynchronize(rt.stream));
        for (const Tensor& t : pads) a.store->release(t.data);
        for (const char* nme : {"q_down", "q_proj", "kv_down", "gate_proj", "k_up", "q_norm", "kv_norm"}) a.drop(nme);
    }

    std::vector<TilingSpec> tilings() const override { return attention_tilings(); }

    Branch forward(Step& st, Tensor x, LayerCache* cache) override {
        Runtime& rt = *st.rt;
        if (!cache || !cache->paged()) fail(IMP_ERROR_INTERNAL, "latent_attention runs against a paged cache");
        const int64_t T = rows(x);
        const ImpCacheView& cv = cache->view;
        Position::Rotary rot{};
        if (!position->rotary(&rot)) fail(IMP_ERROR_INTERNAL, "latent_attention needs rotary tables");
        const int dt = rt.dtype == F32 ? 0 : 1;
        Tensor proj = rt.empty(T, rows(w_down));
        linear(rt, proj, x, w_down);
        const int64_t q_cols = Q > 0 ? Q : (int64_t)H * (D + R);
        Tensor cq{}, q;
        if (Q > 0) {
            // the norms first: the query's product reads the normalised latent
            cq = rt.empty(T, Q);
            prepare(st, proj, Q, cq, Tensor{}, Tensor{}, rot, cv);
            q = rt.empty(T, (int64_t)H * (D + R));
            linear(rt, q, cq, w_uq);
        } else {
            q = col_slice(proj, 0, q_cols);
        }
        Tensor q_lat = rt.empty(T, (int64_t)H * L);
        rt.launches += 1;
        check_launch(imp_grouped_gemm(q_lat.data, q_lat.stride0, L, q.data, q.stride0, D + R, nullptr, w_ukT.data, nullptr, (int64_t)C * D, D, nullptr,
                                      (int)T, C, D, H, 0, dt, rt.stream),
                     "grouped_gemm (latent query)");
        if (Q > 0) {
            ++rt.launches;
            check_launch(imp_latent_query_rope(q.data, q.stride0, (int)T, H, D, R, q_lat.data, q_lat.stride0, C, rot.cos, rot.sin, rot.rot_dim,
                                               rot.max_pos, st.view.positions, dt, rt.status, rt.stream),
                         "latent_query_rope");
        } else {
            prepare(st, col_slice(proj, q_cols, C + R), 0, Tensor{}, q, q_lat, rot, cv);
        }
        Tensor attn = rt.empty(T, (int64_t)H * L);
        paged_attention(st, attn, q_lat, g, *cache, tiling_ids);
        Tensor o = rt.empty(T, (int64_t)H * Dv);
        ++rt.launches;
        const Tensor gate = gated ? col_slice(proj, gate_col, (int64_t)H * Dv) : Tensor{};
        check_launch(imp_grouped_gemm_ex(o.data, o.stride0, Dv, attn.data, attn.stride0, L, nullptr, w_uv.data, nullptr, (int64_t)Dv * C, C, nullptr,
                                         (int)T, Dv, C, H, 0, gated ? GROUPED_SIGMOID_GATE : GROUPED_PLAIN, gate.data, gate.stride0, 0, 0.f, dt, rt.stream),
                     "grouped_gemm (values)");
        return linear(rt, rt.empty(T, rows(w_o)), o, w_o, defer_out);
    }
    // Norms and rotations of `down` = [query latent (q_rank) | latent | rotated key part] and the cache write; with `q` also the
    // rotated parts of the heads' queries, behind their latent-space queries in q_lat.
    void prepare(Step& st, const Tensor& down, int q_rank, const Tensor& cq, const Tensor& q, const Tensor& q_lat, const Position::Rotary& rot,
                 const ImpCacheView& cv) {
        Runtime& rt = *st.rt;
        const size_t el = elem_size(rt.dtype);
        ++rt.launches;
        check_launch(imp_latent_prepare_ex(down.data, down.stride0, (int)rows(down), q_rank, C, R, q_rank > 0 ? (const float*)n_q.data : nullptr,
                                           (const float*)n_kv.data, eps, cq.data, cq.stride0, rot.cos, rot.sin, rot.rot_dim, pairing, rot.max_pos,
                                           st.view.positions, st.view.seq_of_token, cv.block_table, cv.bt_stride, st.B(),
                                           cv.writes ? cv.k_pages : nullptr, L, cv.page_size, cv.num_pages,
                                           q.data ? (const char*)q.data + (size_t)D * el : nullptr, q.stride0, D + R,
                                           q_lat.data ? (char*)q_lat.data + (size_t)C * el : nullptr, q_lat.stride0, H, rt.dtype == F32 ? 0 : 1,
                                           rt.status, rt.stream),
                     "latent_prepare");
    }
};

// -------------------------------------------------------------------------------------------------- wkv
// A linear recurrence with a matrix state per head (see csrc/wkv.cu for the formulas): each of r, k, v, the gate and the
// decay reads the input mixed with the previous token's, x + (x_prev - x) * mu_s; r, k, v = W_s mix_s; gate =
// silu(W_g mix_g); decay = exp(-exp(W_2 tanh(W_1 mix_w) + w0)) per head and key channel; the read-out adds a bonus u for
// the current token; each head's result is divided by its root mean square, times a weight, times the gate; then W_o.
// State per request: S (H heads of D x D; 32-bit in the bfloat16 path, 64-bit in the float32 path, whose read-out would
// otherwise lose five digits where a head's sum nearly cancels) and the last input row (float32), zero at the start.
//
// params: hidden_size, num_heads, head_dim, norm_eps, decay_rank (0 or absent: the rows of the checkpoint's W_1).
struct Wkv : Mixer {
    int H, D;
    float eps;
    Tensor w_r, w_k, w_v, w_g, w_1, w_2, w_o, mu, w0, u, out_norm;   // the last four float32

    static TensorSpecs specs(const Json& p) {
        const char* me = "wkv";
        const int64_t d = need_int(p, "hidden_size", me), H = need_int(p, "num_heads", me), D = need_int(p, "head_dim", me),
                      rank = p.get_int("decay_rank", 0);
        if (H <= 0 || D <= 0 || D > imp_wkv_max_head_dim())
            fail(IMP_ERROR_INVALID_MODEL, std::string(me) + ": head_dim must lie in (0, " + std::to_string(imp_wkv_max_head_dim()) + "] and num_heads be positive");
        TensorSpecs s;
        for (const char* n : {"mu_r", "mu_k", "mu_v", "mu_g", "mu_w"}) s.emplace_back(n, TensorSpec{{d}, "vector", "normal"});
        for (const char* n : {"r_proj", "k_proj", "v_proj", "g_proj"}) s.emplace_back(n, TensorSpec{{H * D, d}});
        s.emplace_back("decay_down", TensorSpec{{rank > 0 ? rank : -1, d}});
        s.emplace_back("decay_up", TensorSpec{{H * D, rank > 0 ? rank : -1}});
        s.emplace_back("decay_bias", TensorSpec{{H * D}, "vector", "normal"});
        s.emplace_back("bonus", TensorSpec{{H, D}, "vector", "normal"});
        s.emplace_back("out_norm", TensorSpec{{H * D}, "norm", "one_plus_normal"});
        s.emplace_back("o_proj", TensorSpec{{d, H * D}});
        return s;
    }
    static CacheSpec cache(const Json& p) {
        const char* me = "wkv";
        const int64_t d = need_int(p, "hidden_size", me), H = need_int(p, "num_heads", me), D = need_int(p, "head_dim", me);
        CacheSpec s;
        s.kind = CacheSpec::State;
        // room for S as 64-bit words: the float32 path carries the state in 64-bit (see csrc/wkv.cu), bfloat16 uses half of it
        s.states.push_back(StateTensorSpec{"S", {H, D, 2 * D}, F32});
        s.states.push_back(StateTensorSpec{"prev", {d}, F32});
        return s;
    }

    explicit Wkv(BuildArgs& a) {
        H = (int)need_int(a.params, "num_heads", "wkv");
        D = (int)need_int(a.params, "head_dim", "wkv");
        eps = (float)a.params.get_double("norm_eps", 1e-6);
        Runtime& rt = *a.rt;
        w_r = a.tensor("r_proj"), w_k = a.tensor("k_proj"), w_v = a.tensor("v_proj"), w_g = a.tensor("g_proj");
        w_1 = a.tensor("decay_down"), w_2 = a.tensor("decay_up"), w_o = a.tensor("o_proj");
        if (rows(w_1) != cols(w_2)) fail(IMP_ERROR_INVALID_MODEL, "wkv: the two decay matrices do not share their inner size");
        std::vector<Tensor> mus;
        for (const char* n : {"mu_r", "mu_k", "mu_v", "mu_g", "mu_w"}) {
            Tensor t = a.tensor(n);
            mus.push_back(tensor2d(t.data, t.dtype, 1, numel(t)));
        }
        Tensor m = cat_rows(rt, *a.store, mus);
        mu = to_float32(rt, *a.store, m);
        w0 = to_float32(rt, *a.store, a.tensor("decay_bias"));
        u = to_float32(rt, *a.store, a.tensor("bonus"));
        out_norm = to_float32(rt, *a.store, a.tensor("out_norm"));
        IMP_CUDA(cudaStreamSynchronize(rt.stream));
        a.store->release(m.data);
        for (const char* n : {"mu_r", "mu_k", "mu_v", "mu_g", "mu_w", "decay_bias", "bonus", "out_norm"}) a.drop(n);
    }

    Branch forward(Step& st, Tensor x, LayerCache* cache) override {
        Runtime& rt = *st.rt;
        if (!cache || cache->view.kind != 2 || cache->view.n_states < 2) fail(IMP_ERROR_INTERNAL, "wkv runs against a state cache");
        const int64_t T = rows(x), d = cols(x), HD = (int64_t)H * D;
        const int dt = rt.dtype == F32 ? 0 : 1;
        float* S = (float*)cache->view.states[0].data;
        float* prev = (float*)cache->view.states[1].data;
        Tensor mixes = rt.empty(5 * T, d);
        const bool single = st.decode_only();
        rt.launches += single ? 1 : 2;
        check_launch(imp_wkv_mix(x.data, x.stride0, (const float*)mu.data, prev, st.view.seq_of_token, st.view.q_start, st.view.state_slots, (int)T,
                                 st.B(), (int)d, mixes.data, single ? 1 : 0, dt, rt.status, rt.stream),
                     "wkv_mix");
        auto mix = [&](int s) { return tensor2d((char*)mixes.data + (size_t)s * (size_t)(T * d) * elem_size(mixes.dtype), mixes.dtype, T, d); };
        Tensor r = rt.empty(T, HD), k = rt.empty(T, HD), v = rt.empty(T, HD), gt = rt.empty(T, HD);
        linear(rt, r, mix(0), w_r);
        linear(rt, k, mix(1), w_k);
        linear(rt, v, mix(2), w_v);
        linear(rt, gt, mix(3), w_g);
        Tensor low = rt.empty(T, rows(w_1));
        linear(rt, low, mix(4), w_1);
        Tensor dlog = rt.empty(T, HD, F32);
        float* o = rt.arena->take<float>((size_t)(T * HD));
        Tensor y = rt.empty(T, HD);
        rt.launches += 3;
        check_launch(imp_tanh_inplace(low.data, numel(low), dt, rt.stream), "tanh");
        linear(rt, dlog, low, w_2);
        // an ordinary dependent launch (see csrc/wkv.cu)
        check_launch(imp_wkv_scan(r.data, k.data, v.data, HD, (const float*)dlog.data, (const float*)w0.data, (const float*)u.data, S, o, st.view.q_start,
                                  st.view.state_slots, st.B(), H, D, dt, rt.stream),
                     "wkv_scan");
        check_launch(imp_wkv_output(y.data, o, gt.data, gt.stride0, (const float*)out_norm.data, eps, (int)T, H, D, dt, rt.stream), "wkv_output");
        return linear(rt, rt.empty(T, rows(w_o)), y, w_o, defer_out);
    }
};

// --------------------------------------------------------------------------------------- routed experts
// A mixture of feed-forward experts, gated by default: router logits z = W_r x + b in 32-bit; the `top_k` experts with the largest
// logits are chosen, weighted by the softmax over the chosen logits; expert e is W_down_e (silu(W_gate_e x) * (W_up_e x)).
// Optionally a shared expert of the same form runs for every token and is added times sigmoid(w_sg . x).
// The experts' matrices are stacked at load; a step sorts its (token, choice) pairs by expert on the device and runs two
// products over the sorted list (csrc/grouped_gemm.cu), so its launches do not depend on the routing.
//
// Options: the router without a bias (`router_bias`: false); sigmoid scores, a chosen expert weighing its score times
// `weight_scale`, not renormalised (`scores`: "sigmoid"; default "softmax" as above); experts in `num_groups` equal groups of
// neighbours of which the `keep_groups` best (by the sum of a group's two largest scores) can be chosen from; a shared expert
// that is added as it is (`shared_gate`: false); scores that are the softmax over all experts, a chosen expert weighing its score
// (`scores`: "softmax_all"); a group counted by its largest score instead of the sum of two (`group_score`: "max", the default with
// "softmax_all"; else "top2"); experts without a gate, W_down_e max(W_up_e x, 0)^2 (`expert`: "relu2"; default "swiglu"; no
// shared expert then), or with both products clipped (`expert`: "clipped", `expert_limit`, and `shared_limit` for the shared
// expert; see gated_mlp); with "softmax_all" a learned bias on the choice only (`choice_bias`: tensor, one number per router output,
// the weights are the scores without it) and weights divided by the chosen ones' sum (`renormalise`); `num_identity` more router
// outputs behind the experts' that stand for the identity, x itself.  With `defer_rows` set the chosen experts' rows are handed on
// unsummed (Branch::rows), where there is a shared expert only if `defer_terms` is set as well: its output is the second summand.
//
// params: hidden_size, num_experts, num_identity, top_k, expert_size, shared_size (0: no shared expert), router_bias, scores,
//         weight_scale, choice_bias, renormalise, num_groups, keep_groups, group_score, shared_gate, expert, expert_limit, shared_limit.
struct RoutedExperts : FeedForward {
    int64_t d, E, I, R, top, F, Fs;    // R = E + I router outputs
    bool has_bias = true, has_sgate = true, gated_expert = true;
    int score_mode = 0, n_groups = 0, keep_groups = 0, group_top = 2;
    float weight_scale = 1.f;
    bool renormalise = false;
    GatedAct act{0}, shared_act{0};
    Tensor choice_bias{};              // float32 [R]
    Tensor w_gate, w_up, w_down;       // [E * F, d], [E * F, d], [E * d, F]; or w_gate [E * 2F, d], gate and up rows alternating in runs of 8
    bool interleaved = false;
    Tensor router, router_bias, sg;    // float32
    Tensor w_route{};                  // bfloat16 router rows (and the shared expert's mixing row behind them), padded to a multiple of 16: the
                                       // logits by the tensor-core product
    cudaStream_t side = nullptr;       // steps of single tokens: the shared expert beside the routed ones
    cudaEvent_t fork = nullptr, join = nullptr;
    ~RoutedExperts() override {
        if (side) cudaStreamDestroy(side);
        if (fork) cudaEventDestroy(fork);
        if (join) cudaEventDestroy(join);
    }
    Tensor s_gu, s_down;               // the shared expert
    bool s_interleaved = false;

    static bool gated_kind(const Json& p) {
        const std::string k = p.get_string("expert", "swiglu");
        if (k != "swiglu" && k != "relu2" && k != "clipped")
            fail(IMP_ERROR_INVALID_MODEL, "routed_experts: unknown expert '" + k + "' (known: swiglu, relu2, clipped)");
        return k != "relu2";
    }
    static GatedAct gated_act_of(const Json& p, const char* limit) {
        if (p.get_string("expert", "swiglu") != "clipped") return GatedAct(0);
        const double l = need_double(p, limit, "routed_experts");
        if (!(l > 0)) fail(IMP_ERROR_INVALID_MODEL, std::string("routed_experts: '") + limit + "' must be positive");
        return GatedAct(2, (float)l);
    }
    static TensorSpecs specs(const Json& p) {
        const char* me = "routed_experts";
        const int64_t d = need_int(p, "hidden_size", me), E = need_int(p, "num_experts", me), top = need_int(p, "top_k", me),
                      F = need_int(p, "expert_size", me), Fs = p.get_int("shared_size", 0), I = p.get_int("num_identity", 0), R = E + I;
        if (E <= 0 || I < 0 || top <= 0 || top > R || F <= 0 || Fs < 0)
            fail(IMP_ERROR_INVALID_MODEL, std::string(me) + ": 0 < top_k <= num_experts + num_identity and positive sizes");
        TensorSpecs s;
        s.emplace_back("router", TensorSpec{{R, d}});
        if (p.get_bool("router_bias", true)) s.emplace_back("router_bias", TensorSpec{{R}, "vector", "normal"});
        if (p.get_bool("choice_bias", false)) s.emplace_back("choice_bias", TensorSpec{{R}, "vector", "zeros"});
        const int64_t ng = p.get_int("num_groups", 0), keep = p.get_int("keep_groups", 0);
        if (ng < 0 || (ng > 0 && (E % ng || keep <= 0 || keep > ng || top > keep * (E / ng))))
            fail(IMP_ERROR_INVALID_MODEL, std::string(me) + ": " + std::to_string(ng) + " groups must divide the " + std::to_string(E) + " experts, and the " +
                                              std::to_string(keep) + " kept groups must hold the " + std::to_string(top) + " chosen experts");
        const std::string sc = p.get_string("scores", "softmax");
        if (sc != "softmax" && sc != "sigmoid" && sc != "softmax_all")
            fail(IMP_ERROR_INVALID_MODEL, std::string(me) + ": unknown scores '" + sc + "' (known: softmax, sigmoid, softmax_all)");
        if ((p.get_bool("choice_bias", false) || p.get_bool("renormalise", false)) && (sc != "softmax_all" || ng > 0))
            fail(IMP_ERROR_UNSUPPORTED, std::string(me) + ": choice_bias and renormalise go with scores 'softmax_all' without groups");
        if (I > 0 && ng > 0) fail(IMP_ERROR_UNSUPPORTED, std::string(me) + ": identity experts go without groups");
        const std::string gsc = p.get_string("group_score", sc == "softmax_all" ? "max" : "top2");
        if ((gsc != "max" && gsc != "top2") || (sc == "softmax_all" && gsc != "max"))
            fail(IMP_ERROR_INVALID_MODEL, std::string(me) + ": unknown group_score '" + gsc + "' (known: top2, max; softmax_all goes with max)");
        const bool gated = gated_kind(p);
        if (!gated && Fs > 0) fail(IMP_ERROR_UNSUPPORTED, std::string(me) + ": experts without a gate go without a shared expert");
        for (int64_t e = 0; e < E; ++e) {
            const std::string n = std::to_string(e);
            if (gated) s.emplace_back("gate_" + n, TensorSpec{{F, d}});
            s.emplace_back("up_" + n, TensorSpec{{F, d}});
            s.emplace_back("down_" + n, TensorSpec{{d, F}});
        }
        if (Fs > 0) {
            s.emplace_back("shared_gate", TensorSpec{{Fs, d}});
            s.emplace_back("shared_up", TensorSpec{{Fs, d}});
            s.emplace_back("shared_down", TensorSpec{{d, Fs}});
            if (p.get_bool("shared_gate", true)) s.emplace_back("shared_mix", TensorSpec{{1, d}});
        }
        return s;
    }

    explicit RoutedExperts(BuildArgs& a) {
        const char* me = "routed_experts";
        d = need_int(a.params, "hidden_size", me), E = need_int(a.params, "num_experts", me), top = need_int(a.params, "top_k", me);
        F = need_int(a.params, "expert_size", me), Fs = a.params.get_int("shared_size", 0);
        I = a.params.get_int("num_identity", 0), R = E + I;
        renormalise = a.params.get_bool("renormalise", false);
        act = gated_act_of(a.params, "expert_limit");
        if (Fs > 0) shared_act = gated_act_of(a.params, "shared_limit");
        has_bias = a.params.get_bool("router_bias", true);
        has_sgate = a.params.get_bool("shared_gate", true);
        gated_expert = gated_kind(a.params);
        const std::string sc = a.params.get_string("scores", "softmax");
        score_mode = sc == "sigmoid" ? 1 : sc == "softmax_all" ? 2 : 0;
        group_top = a.params.get_string("group_score", score_mode == 2 ? "max" : "top2") == "max" ? 1 : 2;
        weight_scale = (float)a.params.get_double("weight_scale", 1.0);
        n_groups = (int)a.params.get_int("num_groups", 0);
        keep_groups = (int)a.params.get_int("keep_groups", 0);
        Runtime& rt = *a.rt;
        std::vector<Tensor> gs, us, ds;
        for (int64_t e = 0; e < E; ++e) {
            const std::string n = std::to_string(e);
            if (gated_expert) gs.push_back(a.tensor("gate_" + n));
            us.push_back(a.tensor("up_" + n));
            ds.push_back(a.tensor("down_" + n));
        }
        // bfloat16 and F a multiple of 8: every expert's gate and up rows alternate in runs of 8, the layout of the fused
        // gate-up product, so that an expert with many rows can go to that product (see forward)
        interleaved = gated_expert && F % SWIGLU_INTERLEAVE == 0 && gs[0].dtype == BF16 && us[0].dtype == BF16;
        if (!gated_expert) {
            w_up = cat_rows(rt, *a.store, us);
        } else if (interleaved) {
            std::vector<Tensor> both;
            for (int64_t e = 0; e < E; ++e) both.push_back(interleave_gate_up(rt, *a.store, gs[(size_t)e], us[(size_t)e]));
            w_gate = cat_rows(rt, *a.store, both);
            IMP_CUDA(cudaStreamSynchronize(rt.stream));
            for (const Tensor& t : both) a.store->release(t.data);
        } else {
            w_gate = cat_rows(rt, *a.store, gs);
            w_up = cat_rows(rt, *a.store, us);
        }
        w_down = cat_rows(rt, *a.store, ds);
        router = to_float32(rt, *a.store, a.tensor("router"));
        if (!rt.is_f32() && a.tensor("router").dtype == BF16 && d % 8 == 0 && (!(Fs > 0 && has_sgate) || a.tensor("shared_mix").dtype == BF16)) {
            std::vector<Tensor> in = {a.tensor("router")};
            if (Fs > 0 && has_sgate) in.push_back(a.tensor("shared_mix"));
            int64_t n = 0;
            for (const Tensor& t : in) n += rows(t);
            const int64_t pad = (16 - n % 16) % 16;
            Tensor zeros{};
            if (pad) {
                zeros = a.store->alloc(BF16, {pad, d});
                IMP_CUDA(cudaMemsetAsync(zeros.data, 0, (size_t)numel(zeros) * 2, rt.stream));
                in.push_back(zeros);
            }
            w_route = cat_rows(rt, *a.store, in);
            IMP_CUDA(cudaStreamSynchronize(rt.stream));
            if (pad) a.store->release(zeros.data);
        }
        if (Fs > 0 && env_flag("IMP_B200_PARALLEL_STREAMS", true)) {
            IMP_CUDA(cudaStreamCreateWithFlags(&side, cudaStreamNonBlocking));
            IMP_CUDA(cudaEventCreateWithFlags(&fork, cudaEventDisableTiming));
            IMP_CUDA(cudaEventCreateWithFlags(&join, cudaEventDisableTiming));
        }
        if (has_bias) router_bias = to_float32(rt, *a.store, a.tensor("router_bias"));
        if (a.params.get_bool("choice_bias", false)) choice_bias = to_float32(rt, *a.store, a.tensor("choice_bias"));
        if (Fs > 0) {
            Tensor gate = a.tensor("shared_gate"), up = a.tensor("shared_up");
            s_interleaved = Fs % SWIGLU_INTERLEAVE == 0 && gate.dtype == up.dtype;
            s_gu = s_interleaved ? interleave_gate_up(rt, *a.store, gate, up) : cat_rows(rt, *a.store, {gate, up});
            s_down = a.tensor("shared_down");
            if (has_sgate) sg = to_float32(rt, *a.store, a.tensor("shared_mix"));
        }
        IMP_CUDA(cudaStreamSynchronize(rt.stream));
        for (int64_t e = 0; e < E; ++e) {
            const std::string n = std::to_string(e);
            if (gated_expert) a.drop("gate_" + n);
            a.drop("up_" + n);
            a.drop("down_" + n);
        }
        a.drop("router");
        if (has_bias) a.drop("router_bias");
        if (choice_bias.data) a.drop("choice_bias");
        if (Fs > 0) {
            for (const char* n : {"shared_gate", "shared_up"}) a.drop(n);
            if (has_sgate) a.drop("shared_mix");
        }
    }

    Branch shared_expert(Runtime& rt, const Tensor& x, bool may_defer) {
        const int64_t T = rows(x);
        Tensor sa = rt.empty(T, Fs);
        if (s_interleaved) {
            linear_gated(rt, sa, x, s_gu, shared_act);
        } else {
            Tensor gu = rt.empty(T, 2 * Fs);
            linear(rt, gu, x, s_gu);
            gated_act(rt, sa, gu, 0, shared_act);
        }
        return linear(rt, rt.empty(T, d), sa, s_down, may_defer);
    }

    Branch forward(Step& st, Tensor x) override {
        Runtime& rt = *st.rt;
        const int64_t T = rows(x), P = T * top;
        const int dt = rt.dtype == F32 ? 0 : 1;
        int* idx = rt.arena->take<int>((size_t)P);
        float* wts = rt.arena->take<float>((size_t)P);
        float* gate = rt.arena->take<float>((size_t)T);
        int* seg = rt.arena->take<int>((size_t)E + 1);
        int* row_token = rt.arena->take<int>((size_t)P);
        int* pair_row = rt.arena->take<int>((size_t)P);
        const bool gated = Fs > 0 && has_sgate;
        const bool hand_on = defer_rows && (Fs == 0 || (defer_terms && !gated));
        // the shared expert needs the input alone: in a step of single tokens it runs on a stream of its own beside the rest
        Branch shared{};
        const bool forked = side && st.decode_only() && !st.diag;
        if (forked) {
            const cudaStream_t main = rt.stream;
            IMP_CUDA(cudaEventRecord(fork, main));
            IMP_CUDA(cudaStreamWaitEvent(side, fork, 0));
            rt.stream = side;
            try {
                shared = shared_expert(rt, x, hand_on && defer_out);
            } catch (...) {
                rt.stream = main;
                throw;
            }
            rt.stream = main;
            IMP_CUDA(cudaEventRecord(join, side));
        }
        rt.launches += 5;
        if (w_route.data && contiguous(x)) {
            const int64_t N = rows(w_route);
            Tensor zl = rt.empty(T, N, F32);
            const Branch z = linear(rt, zl, x, w_route, true);
            const int sorts = imp_moe_choose_sorts((int)T, (int)R, (int)E, (int)top, n_groups, choice_bias.data != nullptr);
            rt.launches -= sorts;
            check_launch(imp_moe_choose(z.split() ? z.parts : (const float*)zl.data, N, z.split() ? z.n_splits : 0, T * N, (int)T,
                                        has_bias ? (const float*)router_bias.data : nullptr, (int)R, (int)E, (int)top, idx, wts, gated ? gate : nullptr,
                                        score_mode, n_groups, keep_groups, group_top, weight_scale, (const float*)choice_bias.data, renormalise ? 1 : 0, seg,
                                        row_token, pair_row, rt.stream),
                         "moe_choose");
        } else {
            check_launch(imp_moe_route_ex(x.data, x.stride0, (int)T, (int)d, (const float*)router.data, has_bias ? (const float*)router_bias.data : nullptr, (int)R,
                                          (int)top, gated ? (const float*)sg.data : nullptr, idx, wts, gate, score_mode, n_groups, keep_groups, group_top,
                                          weight_scale, (const float*)choice_bias.data, renormalise ? 1 : 0, dt, rt.stream),
                         "moe_route");
            check_launch(imp_moe_sort(idx, (int)T, (int)top, (int)E, seg, row_token, pair_row, rt.stream), "moe_sort");
        }
        Tensor hid = rt.empty(P, F);
        Tensor y = rt.empty(P, d);
        // Portions of prompts with much work an expert (rows x F x d of 2^31 and more on average): the list's offsets come to
        // the host, and every expert's rows go to the tensor-memory products as a dense matrix (the wait costs one round
        // trip a layer; 2,048 tokens on 16 experts of 4096 x 4096: 1.2 against 2.0 ms a layer; with experts of 1024 x 1024
        // the products' fixed cost loses: 5.9 against 4.0 ms for four layers).  All other steps, and every step that may
        // be captured into a graph, run the two products over groups, whose launches do not depend on the routing.
        cudaStreamCaptureStatus capturing = cudaStreamCaptureStatusNone;
        IMP_CUDA(cudaStreamIsCapturing(rt.stream, &capturing));
        static const double dense_work = [] { const std::string e = env_string("IMP_B200_MOE_DENSE_WORK", ""); return e.empty() ? 2147483648.0 : std::atof(e.c_str()); }();
        const bool tensor_cores = interleaved || (!gated_expert && w_up.dtype == BF16 && w_down.dtype == BF16 && F % 8 == 0 && d % 8 == 0);
        if (tensor_cores && !st.decode_only() && capturing == cudaStreamCaptureStatusNone && dense_work > 0 &&
            (double)P / (double)R * (double)F * (double)d >= dense_work) {
            std::vector<int> hseg((size_t)E + 1);
            IMP_CUDA(cudaMemcpyAsync(hseg.data(), seg, hseg.size() * 4, cudaMemcpyDeviceToHost, rt.stream));
            IMP_CUDA(cudaStreamSynchronize(rt.stream));
            const int64_t listed = hseg[(size_t)E];   // choices that fell on identity experts are not in the list
            Tensor xs = rt.empty(P, d);
            check_launch(imp_gather_rows(xs.data, x.data, x.stride0, row_token, (int)listed, (int)d, dt, rt.stream), "gather_rows");
            const size_t el = elem_size(rt.dtype);
            for (int64_t e = 0; e < E; ++e) {
                const int64_t a0 = hseg[(size_t)e], n = hseg[(size_t)e + 1] - a0;
                if (n <= 0) continue;
                Tensor xe = tensor2d((char*)xs.data + (size_t)(a0 * d) * el, rt.dtype, n, d);
                Tensor ae = tensor2d((char*)hid.data + (size_t)(a0 * F) * el, rt.dtype, n, F);
                Tensor ye = tensor2d((char*)y.data + (size_t)(a0 * d) * el, rt.dtype, n, d);
                Tensor wd = tensor2d((char*)w_down.data + (size_t)(e * d * F) * el, w_down.dtype, d, F);
                if (gated_expert)
                    linear_gated(rt, ae, xe, tensor2d((char*)w_gate.data + (size_t)(e * 2 * F * d) * el, w_gate.dtype, 2 * F, d), act);
                else
                    linear_relu2(rt, ae, xe, tensor2d((char*)w_up.data + (size_t)(e * F * d) * el, w_up.dtype, F, d));
                linear(rt, ye, ae, wd);
            }
        } else {
            if (!gated_expert)
                check_launch(imp_grouped_gemm_ex(hid.data, F, 0, x.data, x.stride0, 0, row_token, w_up.data, nullptr, F * d, d, seg, (int)P, (int)F, (int)d,
                                                 (int)E, 0, GROUPED_RELU2, nullptr, 0, 0, 0.f, dt, rt.stream),
                             "grouped_gemm (experts, up)");
            else
                check_launch(imp_grouped_gemm_ex(hid.data, F, 0, x.data, x.stride0, 0, row_token, w_gate.data, interleaved ? nullptr : w_up.data,
                                                 (interleaved ? 2 : 1) * F * d, d, seg, (int)P, (int)F, (int)d, (int)E, interleaved ? 2 : 1, 0, nullptr, 0,
                                                 act.kind, act.limit, dt, rt.stream),
                             "grouped_gemm (experts, gate and up)");
            check_launch(imp_grouped_gemm(y.data, d, 0, hid.data, F, 0, nullptr, w_down.data, nullptr, d * F, F, seg, (int)P, (int)d, (int)F, (int)E, 0,
                                          dt, rt.stream),
                         "grouped_gemm (experts, down)");
        }
        if (forked) IMP_CUDA(cudaStreamWaitEvent(rt.stream, join, 0));
        else if (Fs > 0) shared = shared_expert(rt, x, hand_on && defer_out);
        Tensor out = rt.empty(T, d);
        if (hand_on) {
            --rt.launches;
            Branch b = Branch::of(out);
            b.rows = RoutedRows{y.data, pair_row, wts, (int)top, x.data, x.stride0};
            b.second.t = shared.t;
            b.second.parts = shared.parts;
            b.second.n_splits = shared.n_splits;
            return b;
        }
        check_launch(imp_moe_combine(out.data, y.data, pair_row, wts, (int)T, (int)top, Fs > 0 ? shared.t.data : nullptr, gated ? gate : nullptr, x.data,
                                     x.stride0, (int)d, dt, rt.stream),
                     "moe_combine");
        return Branch::of(out);
    }
};

// ------------------------------------------------------------------------- pre-norm block with scaled branches
// h += m * s1 (.) mixer(norm1(h));  h += m * s2 (.) ffn(norm2(h)): a constant m and a learned factor per channel for each
// branch.  The factors ride with the branch (Branch::col_scale) and are multiplied in, in 32-bit, by the norm that adds
// the branch into the stream; where the next normaliser cannot do that the branch is scaled before it is handed on.
// Slots: mixer_norm, mixer, and with has_ffn (default true) ffn_norm, feed_forward.  Tensors: mixer_scale [d] and with
// has_ffn ffn_scale [d].  params: hidden_size, residual_mult (default 1), has_ffn.
struct ScaledPreNormBlock : Block {
    Mixer* mixer_;
    FeedForward* ffn = nullptr;
    Norm *norm1, *norm2 = nullptr;
    Tensor s1, s2;   // float32, times residual_mult
    explicit ScaledPreNormBlock(BuildArgs& a) : mixer_(part_cast<Mixer>(a.part("mixer"), "a mixer")), norm1(part_cast<Norm>(a.part("mixer_norm"), "a norm")) {
        const float m = (float)a.params.get_double("residual_mult", 1.0);
        Runtime& rt = *a.rt;
        auto scaled = [&](const char* name) {
            Tensor f = to_float32(rt, *a.store, a.tensor(name));
            check_launch(imp_scaled_sum(f.data, f.data, m, nullptr, 0.f, nullptr, 0.f, 1, (int)numel(f), F32, rt.stream), "scaled_sum");
            return f;
        };
        s1 = scaled("mixer_scale");
        if (a.params.get_bool("has_ffn", true)) {
            ffn = part_cast<FeedForward>(a.part("feed_forward"), "a feed-forward");
            norm2 = part_cast<Norm>(a.part("ffn_norm"), "a norm");
            s2 = scaled("ffn_scale");
        }
        IMP_CUDA(cudaStreamSynchronize(rt.stream));
        a.drop("mixer_scale");
        if (ffn) a.drop("ffn_scale");
    }
    static std::vector<Slot> slots(const Json& p) {
        std::vector<Slot> s = {{"mixer_norm", "norm"}, {"mixer", "mixer"}};
        if (p.get_bool("has_ffn", true)) {
            s.push_back({"ffn_norm", "norm"});
            s.push_back({"feed_forward", "feed_forward"});
        }
        return s;
    }
    static TensorSpecs specs(const Json& p) {
        const int64_t d = need_int(p, "hidden_size", "scaled_prenorm");
        TensorSpecs s;
        s.emplace_back("mixer_scale", TensorSpec{{d}, "norm", "one_plus_normal"});
        if (p.get_bool("has_ffn", true)) s.emplace_back("ffn_scale", TensorSpec{{d}, "norm", "one_plus_normal"});
        return s;
    }
    bool takes_split_sum() const override { return norm1->takes_split_sum(); }
    bool takes_column_scale() const override { return norm1->takes_column_scale(); }
    Mixer* mixer() const override { return mixer_; }
    std::vector<Part*> parts() const override {
        std::vector<Part*> p = {norm1, mixer_};
        if (ffn) {
            p.push_back(norm2);
            p.push_back(ffn);
        }
        return p;
    }
    bool graph_safe() const override {
        for (Part* p : parts())
            if (!p->graph_safe()) return false;
        return true;
    }
    // The branch with its factors: riding along if the one who adds it multiplies them in, applied now otherwise.
    Branch with_scale(Step& st, Branch b, const Tensor& s, bool consumer_takes) const {
        b.col_scale = (const float*)s.data;
        if (consumer_takes) return b;
        return Branch::of(summed(st, b));
    }
    Branch forward(Step& st, Tensor h, const Branch& pending, LayerCache* cache) override {
        Tensor x = norm1->add_norm(st, h, pending);
        mixer_->defer_out = false;
        Branch a = with_scale(st, mixer_->forward(st, x, cache), s1, ffn ? norm2->takes_column_scale() : scale_pending);
        stage(st, "mixer", a);
        if (!ffn) return a;
        x = norm2->add_norm(st, h, a);
        ffn->defer_out = false;
        Branch f = with_scale(st, ffn->forward(st, x), s2, scale_pending);
        stage(st, "feed_forward", f);
        return f;
    }
};

// ------------------------------------------------------------------------------ the stream re-made from two
// h <- W [h ; x0]: one linear map over the stream and the embedding's output side by side, W [d, 2d] with the stream's
// columns first.  What the block before left pending is added first.  No parts; one tensor, `weight`.
// params: hidden_size.
struct StreamReinjectBlock : Block {
    Tensor weight;
    explicit StreamReinjectBlock(BuildArgs& a) : weight(a.tensor("weight")) {}
    static std::vector<Slot> slots(const Json&) { return {}; }
    static TensorSpecs specs(const Json& p) {
        const int64_t d = need_int(p, "hidden_size", "stream_reinject");
        TensorSpecs s;
        s.emplace_back("weight", TensorSpec{{d, 2 * d}});
        return s;
    }
    bool takes_column_scale() const override { return true; }
    bool wants_embedding() const override { return true; }
    std::vector<Part*> parts() const override { return {}; }
    Branch forward(Step& st, Tensor h, const Branch& pending, LayerCache*) override {
        Runtime& rt = *st.rt;
        if (!st.embedding_out.data) fail(IMP_ERROR_INTERNAL, "stream_reinject: the step kept no copy of the embedding's output");
        const int64_t T = rows(h), d = cols(h);
        const Branch b = parts_summed(rt, pending);
        Tensor both = rt.empty(T, 2 * d);
        ++rt.launches;
        check_launch(imp_concat_streams(both.data, (const float*)h.data, b.empty() ? nullptr : b.t.data, b.col_scale, (const float*)st.embedding_out.data,
                                        (int)T, (int)d, rt.dtype == F32 ? 0 : 1, rt.stream),
                     "concat_streams");
        linear(rt, h, both, weight);   // the stream is float32: the product's sums go there unrounded
        stage(st, "reinject", h);
        return Branch();
    }
};

template <typename T> PartClass class_of(TensorSpecs (*specs)(const Json&)) {
    PartClass c;
    if (specs) c.tensor_specs = specs;
    c.create = [](BuildArgs& a) -> Part* { return new T(a); };
    return c;
}

}  // namespace

void register_routed_parts() {
    PartClass norm = class_of<LayerNorm>(nullptr);
    norm.tensor_specs = [](const Json& p) {
        TensorSpecs s;
        s.emplace_back("weight", TensorSpec{{need_int(p, "size", "layernorm")}, "norm", "one_plus_normal"});
        if (p.get_bool("bias", false)) s.emplace_back("bias", TensorSpec{{need_int(p, "size", "layernorm")}, "vector", "normal"});
        return s;
    };
    register_part_class("norm", "layernorm", norm, true);
    PartClass la = class_of<LatentAttention>(&LatentAttention::specs);
    la.cache_spec = &LatentAttention::cache;
    register_part_class("mixer", "latent_attention", la, true);
    PartClass wkv = class_of<Wkv>(&Wkv::specs);
    wkv.cache_spec = &Wkv::cache;
    register_part_class("mixer", "wkv", wkv, true);
    register_part_class("feed_forward", "routed_experts", class_of<RoutedExperts>(&RoutedExperts::specs), true);
    PartClass block = class_of<ScaledPreNormBlock>(&ScaledPreNormBlock::specs);
    block.part_slots = &ScaledPreNormBlock::slots;
    register_part_class("block", "scaled_prenorm", block, true);
    PartClass inject = class_of<StreamReinjectBlock>(&StreamReinjectBlock::specs);
    inject.part_slots = &StreamReinjectBlock::slots;
    register_part_class("block", "stream_reinject", inject, true);
}

}  // namespace imp
