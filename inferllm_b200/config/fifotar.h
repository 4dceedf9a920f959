// Typed configuration of the Fifotar decoder, read from its config.json keys.
//
// A Fifotar model lists its layers one by one: `layers[i]` has `type` ("delta": a gated delta rule with one decay per head
// over per-sequence state; "latent_attention": attention through a query latent and a key/value latent with a rotated key
// part that all heads share; "attention": attention without positions inside chunks of the sequence, with capped scores,
// a sink of score 0 and an element-wise gate), `mixer` (the mixer's sizes and constants) and `mlp` ({"kind": "dense",
// "ff": n, "limit": L}, or null for a layer without a feed-forward).  Beside the list: `width`, `vocab`, `norm.eps`,
// `embedding.scale`, `residual_mult` (the factor on every sublayer's normed output), `logit_softcap` and optionally
// `max_positions` (the longest sequence; 131072 if not given).  Every layer norms each sublayer's input and output (RMS
// norms); the output matrix is the embedding table.  What the mixers are is said where they are mapped to parts
// (config/fifotar.cpp).
#pragma once
#include "config/config.h"

namespace illm {

struct FifotarConfig : ArchConfig {
    Json raw;                    // the config.json object as it was read (to_json gives it back)
    long long width = 0, vocab = 0, max_positions = 131072;
    double norm_eps = 1e-6, embedding_scale = 1.0, residual_mult = 1.0, logit_softcap = 0.0;

    static std::unique_ptr<ArchConfig> from_json(const Json& d);
    std::string architecture() const override { return "Fifotar"; }
    Json to_json() const override { return raw; }
    ModelSpec model_spec() const override;
};

}  // namespace illm
