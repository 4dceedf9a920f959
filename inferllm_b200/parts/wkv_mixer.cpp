// A time-mixing recurrence over a per-sequence state: the mixer "wkv".
//
//     m_s = x_t + (x_(t-1) - x_t) * mu_s                      for s = r, k, v, g, w (x_(-1) = 0)
//     r, k, v = W_r m_r, W_k m_k, W_v m_v  [heads x d];   gate = silu(W_g m_g)
//     w = exp(-exp(W_w2 tanh(W_w1 m_w) + w0))                  per head and key channel, in (0, 1)
//     o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t;   S_t = diag(w_t) S_(t-1) + k_t v_t^T           (per head, float32)
//     y = W_o ( o / rms(o) per head * norm * gate )
//
// The mixer reads the float32 stream itself (reads_stream): the blends are made from it and rounded once.  Everything from the
// float32 projections to the normed, gated row is float32.  Cache entry: S [heads, d, d] and the sequence's last row x, float32,
// zero when a sequence starts.  The inner size of the decay's low-rank map is the tensors'.  Tensors: `names` gives "r", "k",
// "v", "gate", "o", "norm", "bonus" (u), "w1", "w2", "w0", and the blends' prefix "mu", followed by r, k, v, w and, for the
// gate's, "mu_gate".
#include <cmath>

#include "parts/parts.h"

namespace illm {

namespace {

struct WkvMixer : Mixer {
    long long hidden;
    int n_heads, head_dim, rank = 0, rank_rows = 0;      // rank_rows: the rank in whole pieces of eight rows (the rest zeros)
    float norm_eps;
    bool out_f32;
    std::map<std::string, std::string> names;
    DeviceBuffer mu_buf, in_buf;
    Mat w_in;                   // rows: r, k, v, gate, then the decay's inner map
    OwnedMat w2, w0, u, norm_w, w_o;

    WkvMixer(const PartSpec& s, Runtime* rt)
            : Mixer(s, rt), hidden(s.get_int("hidden_size")), n_heads((int)s.get_int("n_heads")), head_dim((int)s.get_int("head_dim")),
              norm_eps((float)s.get_double("norm_eps", 1e-6)), out_f32(s.get_string("output_dtype", "compute") == "float32") {
        if (hidden <= 0 || n_heads <= 0 || head_dim <= 0) throw ConfigError("wkv: sizes must be positive");
        names = {{"r", "r_proj.weight"}, {"k", "k_proj.weight"}, {"v", "v_proj.weight"}, {"gate", "g_proj.weight"}, {"o", "o_proj.weight"}, {"mu", "mu."},
                 {"mu_gate", "g"}, {"w1", "w1"}, {"w2", "w2"}, {"w0", "w0"}, {"bonus", "u"}, {"norm", "norm.weight"}};
        if (s.has("names"))
            for (auto& m : s.params.at("names").members()) names[m.first] = m.second.as_string();
        if (rt && !ops::wkv_supported(head_dim, head_dim)) throw ConfigError("wkv: heads of more than 1024 channels are beyond the kernel");
    }
    bool graph_safe() const override { return true; }
    bool pad_safe() const override { return false; }
    bool reads_stream() const override { return true; }
    long long width() const { return (long long)n_heads * head_dim; }
    long long prev_off() const { return (width() * head_dim + 3) / 4 * 4; }
    CacheRequest cache_request() const override { return CacheRequest::state({(prev_off() + hidden + 3) / 4 * 4}, DType::F32); }
    std::string blend(const char* role) const { return names.at("mu") + (role[0] == 'g' ? names.at("mu_gate") : std::string(role)); }
    TensorDecls tensors() const override {
        auto nm = [&](const char* r) { return names.at(r); };
        const long long n = width();
        TensorDecls d;
        for (const char* s : {"r", "k", "v", "g", "w"}) d.push_back({blend(s), TensorDecl{{hidden}}});
        for (const char* s : {"r", "k", "v", "gate"}) d.push_back({nm(s), TensorDecl{{n, hidden}}});
        const long long inner = spec.get_int("decay_rank", -1);
        d.push_back({nm("w1"), TensorDecl{{inner, hidden}}});
        d.push_back({nm("w2"), TensorDecl{{n, inner}}});
        d.push_back({nm("w0"), TensorDecl{{n}}});
        d.push_back({nm("bonus"), TensorDecl{{(long long)n_heads, (long long)head_dim}}});
        d.push_back({nm("norm"), TensorDecl{{n}, "norm"}});
        d.push_back({nm("o"), TensorDecl{{hidden, n}}});
        return d;
    }
    void load(TensorSource& src) override {
        const size_t es = dtype_size(rt->dtype);
        const long long n = width();
        const std::vector<long long> s1 = src.shape(names.at("w1")), s2 = src.shape(names.at("w2"));
        if (s1.size() != 2 || s2.size() != 2 || s1[0] != s2[1] || s1[0] <= 0) throw WeightError("wkv: the two matrices of the decay's map do not fit together");
        rank = (int)s1[0];
        rank_rows = (rank + 7) / 8 * 8;
        mu_buf = DeviceBuffer(rt->dev, (size_t)5 * hidden * sizeof(float), "a mixer's blends");
        int i = 0;
        for (const char* s : {"r", "k", "v", "g", "w"}) src.fetch_into(blend(s), (float*)mu_buf.get() + (size_t)(i++) * hidden, DType::F32);
        const long long rows = 4 * n + rank_rows;
        in_buf = DeviceBuffer(rt->dev, (size_t)rows * hidden * es, "the stacked projections of a time-mixing layer");
        w_in = Mat{in_buf.get(), rows, hidden, rt->dtype, rows};
        check_cuda(cudaMemsetAsync(in_buf.get(), 0, in_buf.bytes(), rt->dev->stream()), "clearing the stacked projections");
        i = 0;
        for (const char* s : {"r", "k", "v", "gate"}) src.fetch_into(names.at(s), (char*)in_buf.get() + (size_t)(i++) * n * hidden * es, rt->dtype);
        src.fetch_into(names.at("w1"), (char*)in_buf.get() + (size_t)4 * n * hidden * es, rt->dtype);
        w2 = fetch_owned(rt, src, names.at("w2"), rt->dtype, "the outer matrix of a decay's map");
        w0 = fetch_owned(rt, src, names.at("w0"), DType::F32, "a decay's offset");
        u = fetch_owned(rt, src, names.at("bonus"), DType::F32, "a bonus");
        norm_w = fetch_owned(rt, src, names.at("norm"), DType::F32, "a time-mixing layer's norm weight");
        w_o = fetch_owned(rt, src, names.at("o"), rt->dtype, "the output matrix of a time-mixing layer");
    }
    MatOrPartials forward(const Mat& x, const StepContext& ctx, const CacheView& cache, bool writes, bool may_defer) override {
        if (cache.kind != CacheView::State) throw EngineError("wkv: the layer's cache entry holds no state");
        if (!writes) throw EngineError("wkv: the state belongs to one layer");
        Device& dev = *rt->dev;
        const int n = (int)width();
        Mat xf = ops::cast(dev, x, DType::F32);
        long long group_rows = 0;
        Mat mixed = ops::token_mix(dev, xf, (const float*)mu_buf.get(), 5, ctx, cache.st, prev_off(), rt->dtype, &group_rows);
        ops::WkvScan p;
        p.r_off = 0;
        p.k_off = n;
        p.v_off = 2 * n;
        p.z_off = 4 * n;
        p.rank = rank;
        p.n_heads = n_heads;
        p.head_dim = p.v_head_dim = head_dim;
        p.w2 = &w2.m;
        p.w0 = (const float*)w0.m.p;
        p.u = (const float*)u.m.p;
        p.in_order = rt->is_f32();      // the float32 mode gives the same bits however a prompt is cut
        const bool one = ctx.is_decode && !rt->is_f32() && ops::wkv_step_supported(p, cache.st);
        MatOrPartials y = ops::group_linear(dev, rt->gemm, mixed, group_rows, xf.rows, w_in, {n, n, n, n, rank_rows}, one);
        if (one)        // one token per sequence: everything up to the gated row in one kernel, which also adds up the slices
            return ops::linear(dev, rt->gemm, ops::wkv_step(dev, y, p, 3 * n, (const float*)norm_w.m.p, norm_eps, ctx, cache.st), w_o.m,
                               out_f32 ? DType::F32 : rt->dtype, may_defer);
        Mat o = ops::wkv_scan(dev, y.m, p, ctx, cache.st);
        Mat g = ops::group_norm_gate(dev, o, head_dim, (const float*)norm_w.m.p, norm_eps, (const float*)y.m.p + 3 * n, (int)y.m.cols, 1, rt->dtype);
        return ops::linear(dev, rt->gemm, g, w_o.m, out_f32 ? DType::F32 : rt->dtype, may_defer);
    }
};

}  // namespace

void register_wkv_parts(std::map<std::string, PartFactory<Mixer>>& mixers) {
    mixers["wkv"] = [](const PartSpec& s, Runtime* rt) { return std::unique_ptr<Mixer>(new WkvMixer(s, rt)); };
}

}  // namespace illm
