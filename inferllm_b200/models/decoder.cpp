#include "models/decoder.h"

#include "cache/cache.h"

namespace illm {

static std::string role_name(const LayerSpec& ls, const std::string& role) {
    auto it = ls.names.find(role);
    if (it == ls.names.end()) throw ConfigError("layer '" + ls.prefix + "': no tensor-name prefix for the role '" + role + "'");
    return it->second;
}

DecoderModel::DecoderModel(const ModelSpec& s, Runtime* runtime) : spec(s), rt(runtime) {
    spec.validate();
    embedding_ = build_embedding(spec.embedding, rt);
    for (const LayerSpec& ls : spec.layers) {
        const BlockKind& kind = lookup_block(ls.block);
        Layer l;
        l.mixer = build_mixer(ls.mixer, rt);
        if (!ls.ffn.kind.empty()) l.ffn = build_feed_forward(ls.ffn, rt);      // a layer may have no feed-forward
        l.block = kind.make();
        l.block->mixer = l.mixer.get();
        l.block->ffn = l.ffn.get();
        for (const std::string& role : kind.norm_roles) {
            auto it = ls.norms.find(role);
            if (it == ls.norms.end())
                throw ConfigError("layer '" + ls.prefix + "': the block arrangement '" + ls.block + "' needs a norm for the role '" + role + "'");
            l.norms[role] = build_norm(it->second, rt);
            l.block->norms[role] = l.norms[role].get();
        }
        layers_.push_back(std::move(l));
    }
    final_norm_ = build_norm(spec.final_norm, rt);
    head_ = build_head(spec.head, rt);
    // "add_embedding" is no part: the embedding output itself is added to the stream
    if (!spec.reentry.kind.empty() && spec.reentry.kind != kReentryAddEmbedding) reentry_ = build_feed_forward(spec.reentry, rt);
}

std::vector<std::pair<std::string, Part*>> DecoderModel::owners() const {
    std::vector<std::pair<std::string, Part*>> out;
    out.emplace_back(spec.embedding.get_string("name", ""), embedding_.get());
    for (size_t i = 0; i < layers_.size(); i++) {
        const LayerSpec& ls = spec.layers[i];
        out.emplace_back(ls.prefix + role_name(ls, "mixer"), layers_[i].mixer.get());
        if (layers_[i].ffn) out.emplace_back(ls.prefix + role_name(ls, "ffn"), layers_[i].ffn.get());
        for (auto& n : layers_[i].norms) out.emplace_back(ls.prefix + role_name(ls, n.first), n.second.get());
    }
    if (reentry_) out.emplace_back(spec.reentry.get_string("name", ""), reentry_.get());
    out.emplace_back(spec.final_norm.get_string("name", ""), final_norm_.get());
    out.emplace_back(spec.head.get_string("name", ""), head_.get());
    return out;
}

std::vector<std::pair<std::string, TensorDecl>> DecoderModel::tensor_decls(bool include_optional) const {
    std::vector<std::pair<std::string, TensorDecl>> decls;
    for (auto& o : owners())
        for (auto& d : o.second->tensors())
            if (include_optional || !d.second.optional) decls.emplace_back(o.first + d.first, d.second);
    return decls;
}

void DecoderModel::load_tensors(const std::function<std::unique_ptr<TensorSource>(const std::string&)>& open) {
    for (auto& o : owners()) {
        if (o.second->tensors().empty()) continue;
        std::unique_ptr<TensorSource> src = open(o.first);
        o.second->load(*src);
    }
    if (head_->tied()) head_->tie(*embedding_);
}

std::map<int, CacheRequest> DecoderModel::cache_requests() const {
    std::map<int, CacheRequest> out;
    for (const ScheduleEntry& e : spec.schedule)
        if (e.writes) {
            out[e.cache] = layers_[(size_t)e.layer].mixer->cache_request();
            const CacheRequest aux = layers_[(size_t)e.layer].mixer->aux_cache_request();
            if (aux.kind == CacheRequest::FixedState) out[kAuxCacheEntryBase + e.cache] = aux;
            else if (aux.kind != CacheRequest::None) throw ConfigError("a mixer's second cache entry must be fixed state");
        }
    // an entry that other layers read too keeps what the farthest-reaching of them sees (those mask for themselves)
    for (const ScheduleEntry& e : spec.schedule) {
        if (e.writes) continue;
        const Mixer::Reach r = layers_[(size_t)e.layer].mixer->reach();
        auto it = out.find(e.cache);
        if (r.known && it != out.end() && it->second.kind == CacheRequest::PagedKV) it->second = it->second.reaching(r.window, r.chunk);
    }
    const CacheRequest er = embedding_->cache_request();
    if (er.kind != CacheRequest::None) out[kEmbeddingCacheEntry] = er;
    return out;
}

Mat DecoderModel::forward(const StepContext& ctx, const SequenceCache& cache, const std::vector<const int*>& tables_dev) {
    Device& dev = *rt->dev;
    ctx.kept.clear();
    ResidualStream stream;
    if (cache.kind_of(kEmbeddingCacheEntry) == SequenceCache::State) {
        CacheView ev;
        ev.kind = CacheView::State;
        ev.st = cache.state_view(kEmbeddingCacheEntry, ctx.slots);
        stream = embedding_->forward_with_state(ctx, ev);
    } else {
        stream = embedding_->forward(ctx);
    }
    Mat x0;      // the embedding output, kept for the entries that re-enter the stream
    const bool reenters = !spec.reentry.kind.empty();
    if (reenters) {
        stream.flush();
        x0 = stream.x;
        x0.p = dev.alloc(x0.bytes());
        check_cuda(cudaMemcpyAsync(x0.p, stream.x.p, x0.bytes(), cudaMemcpyDeviceToDevice, dev.stream()), "keeping the embedding output");
    }
    int turn = 0;
    for (const ScheduleEntry& e : spec.schedule) {
        // the layers' activations take turns in two lanes of the step arena: what a layer leaves for the
        // next one (its last output, pending in the stream) is read before this lane's turn comes again
        dev.set_lane(1 + (turn++ & 1), true);
        if (e.reenter && !reentry_) {
            // x <- x + x0, in float32
            stream.flush();
            MatOrPartials again;
            again.m = x0;
            ops::residual_add(dev, stream.x, again);
        } else if (e.reenter) {
            // x <- W [x; x0]; the result goes back into the stream's own rows, which outlive the lanes
            stream.flush();
            MatOrPartials y = reentry_->forward(ops::join_rows(dev, stream.x, x0, rt->dtype), ctx, false);
            if (y.m.dtype != DType::F32 || y.m.rows != stream.x.rows || y.m.cols != stream.x.cols)
                throw EngineError("the re-entry map must give float32 rows of the stream's width");
            check_cuda(cudaMemcpyAsync(stream.x.p, y.m.p, stream.x.bytes(), cudaMemcpyDeviceToDevice, dev.stream()), "re-entering the stream");
        }
        CacheView view;
        switch (cache.kind_of(e.cache)) {
            case SequenceCache::KV:
                view.kind = CacheView::KV;
                view.kv = cache.kv_view(e.cache, tables_dev[(size_t)cache.group_of(e.cache)]);
                view.kv.writes = e.writes;
                break;
            case SequenceCache::State:
                view.kind = CacheView::State;
                view.st = cache.state_view(e.cache, ctx.slots);
                break;
            default: break;
        }
        if (cache.kind_of(kAuxCacheEntryBase + e.cache) == SequenceCache::State) {
            view.has_aux = true;
            view.aux = cache.state_view(kAuxCacheEntryBase + e.cache, ctx.slots);
        }
        layers_[(size_t)e.layer].block->forward(stream, ctx, view, e.writes);
    }
    dev.set_lane(0, false);
    if (ctx.K == 0) {
        Mat none;
        none.cols = spec.vocab_size;
        none.dtype = DType::F32;
        return none;
    }
    Mat y = final_norm_->forward(stream, ctx.want_rows, ctx.K);
    return head_->forward(y, ctx);
}

bool DecoderModel::graph_safe() const {
    for (const Layer& l : layers_)
        if (!l.mixer->graph_safe() || (l.ffn && !l.ffn->graph_safe())) return false;
    return true;
}
bool DecoderModel::pad_safe() const {
    if (!graph_safe() || !embedding_->pad_safe()) return false;
    for (const Layer& l : layers_)
        if (!l.mixer->pad_safe()) return false;
    return true;
}

}  // namespace illm
