// Part kinds: a norm that computes no statistics, a token embedding with a second table of hashed token pairs (and the state that
// takes), and a block whose mixer and feed-forward read one norm's output side by side.  Every size and constant is a
// parameter; no kind knows which model it is in.
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

// --------------------------------------------------------------------------------------------- dynamic tanh
// y = tanh(alpha x) * w + b with a scalar alpha: nothing is summed over a row, so the kernel that adds a branch into the stream and
// normalises it is element by element (csrc/dynamic_tanh.cu).  It takes branches as they come: unsummed parts of a product, two
// summands with a constant factor, rows of routed experts.
// params: size.  Tensors: weight, bias [size], alpha (a scalar).
struct DynamicTanh : Norm {
    Tensor weight, bias, alpha;   // alpha float32
    static TensorSpecs specs(const Json& p) {
        const int64_t d = need_int(p, "size", "dynamic_tanh");
        TensorSpecs s;
        s.emplace_back("weight", TensorSpec{{d}, "norm", "one_plus_normal"});
        s.emplace_back("bias", TensorSpec{{d}, "vector", "normal"});
        s.emplace_back("alpha", TensorSpec{{}, "norm", "one_plus_normal"});
        return s;
    }
    explicit DynamicTanh(BuildArgs& a) : weight(a.tensor("weight")), bias(a.tensor("bias")) {
        if (bias.dtype != weight.dtype || numel(bias) != numel(weight)) fail(IMP_ERROR_INVALID_MODEL, "dynamic_tanh: weight and bias must agree in type and size");
        alpha = to_float32(*a.rt, *a.store, a.tensor("alpha"));
        IMP_CUDA(cudaStreamSynchronize(a.rt->stream));
        a.drop("alpha");
    }
    bool takes_split_sum() const override { return true; }
    bool takes_branch_pair() const override { return true; }
    Tensor add_norm(Step& st, Tensor h, const Branch& branch, const int32_t* rows_idx, int n_rows) override {
        Runtime& rt = *st.rt;
        const int64_t n = rows_idx ? n_rows : rows(h);
        const int d = (int)cols(h);
        Tensor out = rt.empty(n, d, -1, /*step=*/rows_idx != nullptr);
        if (h.dtype != F32 || !contiguous(h) || numel(weight) != d) fail(IMP_ERROR_INVALID_ARG, "dynamic_tanh: the stream must be dense float32 [T, d], the weight [d]");
        Branch b = branch;
        const bool far_input = (b.rows.input && b.rows.input_ld != d) || (b.second.rows.input && b.second.rows.input_ld != d);
        if (b.col_scale || b.own_norm.weight || b.bias || far_input) b = Branch::of(summed(rt, b));
        for (const Tensor* t : {&b.t, &b.second.t})
            if (t->data && (rows(*t) != rows(h) || cols(*t) != d || t->dtype != out.dtype || !contiguous(*t)))
                fail(IMP_ERROR_INVALID_ARG, "dynamic_tanh: a branch must be dense, of the stream's shape and the output's type");
        const ImpBranchTerm first = branch_term(b.t, b.parts, b.n_splits, b.rows), second = branch_term(b.second.t, b.second.parts, b.second.n_splits, b.second.rows);
        ++rt.launches;
        rt.split_norm_calls += b.parts || b.second.parts;
        check_launch(imp_add_dyt((float*)h.data, b.mult, &first, &second, (const float*)alpha.data, weight.data, bias.data, out.data, rows_idx, (int)rows(h),
                                 (int)n, d, out.dtype, weight.dtype, rt.stream),
                     "add_dyt");
        return out;
    }
};

// ------------------------------------------------------------------------------- embedding with a table of token pairs
// h[t] = E[id] * scale + P[(prev * mul_prev + id * mul_cur) mod buckets], prev the token before; a sequence's first token takes
// P's last row, number `buckets`.  State per request: the last token (int32).
// params: vocab_size, hidden_size, buckets, mul_prev, mul_cur, scale (default 1).  Tensors: weight, bigram [buckets + 1, hidden_size].
struct BigramEmbedding : Embedding {
    Tensor weight, bigram;
    int64_t buckets, mul_prev, mul_cur;   // the multipliers modulo the buckets
    float scale;
    static TensorSpecs specs(const Json& p) {
        const char* me = "bigram_embedding";
        const int64_t d = need_int(p, "hidden_size", me), n = need_int(p, "buckets", me);
        if (n <= 0 || n >= INT32_MAX) fail(IMP_ERROR_INVALID_MODEL, std::string(me) + ": 'buckets' must be positive");
        TensorSpecs s;
        s.emplace_back("weight", TensorSpec{{need_int(p, "vocab_size", me), d}});
        s.emplace_back("bigram", TensorSpec{{n + 1, d}});
        return s;
    }
    static CacheSpec cache(const Json&) {
        CacheSpec s;
        s.kind = CacheSpec::State;
        s.states.push_back(StateTensorSpec{"last_token", {1}, I32});
        return s;
    }
    explicit BigramEmbedding(BuildArgs& a) : weight(a.tensor("weight")), bigram(a.tensor("bigram")), scale((float)a.params.get_double("scale", 1.0)) {
        const char* me = "bigram_embedding";
        buckets = need_int(a.params, "buckets", me);
        auto reduced = [&](const char* key) { return (need_int(a.params, key, me) % buckets + buckets) % buckets; };
        mul_prev = reduced("mul_prev");
        mul_cur = reduced("mul_cur");
        if (weight.dtype != bigram.dtype) fail(IMP_ERROR_INVALID_MODEL, std::string(me) + ": the two tables must be of one type");
    }
    Tensor forward(Step& st, LayerCache* cache) override {
        Runtime& rt = *st.rt;
        if (!cache || cache->view.kind != 2 || cache->view.n_states < 1) fail(IMP_ERROR_INTERNAL, "bigram_embedding runs against a state cache");
        Tensor out = rt.empty(st.T(), cols(weight), F32, /*step=*/true);
        ++rt.launches;
        check_launch(imp_bigram_embedding((float*)out.data, weight.data, bigram.data, st.view.token_ids, st.view.positions, st.view.seq_of_token,
                                          st.view.q_start, st.view.state_slots, (int32_t*)cache->view.states[0].data, st.T(), st.B(), (int)cols(weight),
                                          (int)rows(weight), (int)buckets, mul_prev, mul_cur, weight.dtype, scale, rt.status, rt.stream),
                     "bigram_embedding");
        return out;
    }
};

// ------------------------------------------------------------------------------------ sublayers side by side
// x = norm(h);  h += m (mixer(x) + ffn(x)): one norm, read by both sublayers.  The two outputs travel as the two summands of one
// branch, unsummed parts and routed rows included, to the norm that adds them; where that norm takes plain branches only, the sum
// is worked out first.  In steps of single tokens, where each sublayer is a chain of short launches, the feed-forward runs on a
// stream of its own beside the mixer (a fork after the norm, a join before the branch is handed on; a captured graph has the same
// two paths); IMP_B200_PARALLEL_STREAMS=0 runs them one after the other.
// Slots: norm, mixer, and with has_ffn (default true) feed_forward.  params: residual_mult (default 1), has_ffn.
struct ParallelBlock : Block {
    Norm* norm;
    Mixer* mixer_;
    FeedForward* ffn = nullptr;
    float mult;
    cudaStream_t side = nullptr;
    cudaEvent_t fork = nullptr, join = nullptr;
    ~ParallelBlock() override {
        if (side) cudaStreamDestroy(side);
        if (fork) cudaEventDestroy(fork);
        if (join) cudaEventDestroy(join);
    }
    explicit ParallelBlock(BuildArgs& a)
        : norm(part_cast<Norm>(a.part("norm"), "a norm")), mixer_(part_cast<Mixer>(a.part("mixer"), "a mixer")),
          mult((float)a.params.get_double("residual_mult", 1.0)) {
        if (!a.params.get_bool("has_ffn", true)) return;
        ffn = part_cast<FeedForward>(a.part("feed_forward"), "a feed-forward");
        if (mixer_->graph_safe() && ffn->graph_safe() && env_flag("IMP_B200_PARALLEL_STREAMS", true)) {
            IMP_CUDA(cudaStreamCreateWithFlags(&side, cudaStreamNonBlocking));
            IMP_CUDA(cudaEventCreateWithFlags(&fork, cudaEventDisableTiming));
            IMP_CUDA(cudaEventCreateWithFlags(&join, cudaEventDisableTiming));
        }
    }
    // The feed-forward on the side stream, from what the step's stream holds so far; `join` stands behind it.
    Branch forked_ffn(Step& st, const Tensor& x) {
        Runtime& rt = *st.rt;
        const cudaStream_t main = rt.stream;
        IMP_CUDA(cudaEventRecord(fork, main));
        IMP_CUDA(cudaStreamWaitEvent(side, fork, 0));
        rt.stream = side;
        Branch f;
        try {
            f = ffn->forward(st, x);
        } catch (...) {
            rt.stream = main;
            throw;
        }
        rt.stream = main;
        IMP_CUDA(cudaEventRecord(join, side));
        return f;
    }
    static std::vector<Slot> slots(const Json& p) {
        std::vector<Slot> s = {{"norm", "norm"}, {"mixer", "mixer"}};
        if (p.get_bool("has_ffn", true)) s.push_back({"feed_forward", "feed_forward"});
        return s;
    }
    bool takes_split_sum() const override { return norm->takes_split_sum(); }
    bool takes_column_scale() const override { return norm->takes_column_scale(); }
    bool takes_normed_branch() const override { return norm->takes_normed_branch(); }
    bool takes_branch_pair() const override { return norm->takes_branch_pair(); }
    Mixer* mixer() const override { return mixer_; }
    std::vector<Part*> parts() const override {
        std::vector<Part*> p = {norm, mixer_};
        if (ffn) p.push_back(ffn);
        return p;
    }
    bool graph_safe() const override {
        for (Part* p : parts())
            if (!p->graph_safe()) return false;
        return true;
    }
    Branch forward(Step& st, Tensor h, const Branch& pending, LayerCache* cache) override {
        Tensor x = norm->add_norm(st, h, pending);
        mixer_->defer_out = defer_pending && pair_pending;
        if (ffn) {
            ffn->defer_out = defer_pending && pair_pending;
            ffn->defer_rows = pair_pending;
        }
        const bool forked = ffn && side && st.decode_only() && !st.diag;
        Branch f;
        if (forked) f = forked_ffn(st, x);
        Branch out = mixer_->forward(st, x, cache);
        stage(st, "mixer", out);
        if (ffn) {
            if (forked) IMP_CUDA(cudaStreamWaitEvent(st.rt->stream, join, 0));
            else f = ffn->forward(st, x);
            stage(st, "feed_forward", f.rows.y ? Branch() : f);
            if (f.col_scale || f.own_norm.weight || f.mult != 1.f || !f.second.empty() || f.bias) fail(IMP_ERROR_INTERNAL, "parallel: a feed-forward returns a plain branch");
            out.second.t = f.t;
            out.second.parts = f.parts;
            out.second.n_splits = f.n_splits;
            out.second.rows = f.rows;
        }
        out.mult = mult;
        return pair_pending ? out : Branch::of(summed(st, out));
    }
};

template <typename T> PartClass class_of(TensorSpecs (*specs)(const Json&)) {
    PartClass c;
    if (specs) c.tensor_specs = specs;
    c.create = [](BuildArgs& a) -> Part* { return new T(a); };
    return c;
}

}  // namespace

void register_parallel_parts() {
    register_part_class("norm", "dynamic_tanh", class_of<DynamicTanh>(&DynamicTanh::specs), true);
    PartClass em = class_of<BigramEmbedding>(&BigramEmbedding::specs);
    em.cache_spec = &BigramEmbedding::cache;
    register_part_class("embedding", "bigram_embedding", em, true);
    PartClass block = class_of<ParallelBlock>(nullptr);
    block.part_slots = &ParallelBlock::slots;
    register_part_class("block", "parallel", block, true);
}

}  // namespace imp
