// Typed configuration of the Zeluzen decoder, read from its config.json keys.
//
// A Zeluzen model lists its layers one by one: `layers[i]` has `type` ("wkv": a time-mixing recurrence with a decay per head
// and key channel over per-sequence state; "attention": softmax attention inside chunks of the sequence with normed and
// rotated queries and keys, optionally on another layer's keys and values), `mixer` (the mixer's sizes and constants) and
// `mlp` ({"kind": "dense", "ff": n}, {"kind": "moe", "expert": {"ff": n}, "router": {"experts": E, "identity": I, "top": k}},
// or null for a layer without a feed-forward).  Beside the list: `width`, `vocab`, `norm.eps` and optionally `max_positions`
// (the longest sequence; 131072 if not given).  The embedding's row is normed; every sublayer reads the stream as it is and
// its output is normed on the way into it (RMS norms); the output matrix is a tensor of its own.  What the mixers are is
// said where they are mapped to parts (config/zeluzen.cpp).
#pragma once
#include "config/config.h"

namespace illm {

struct ZeluzenConfig : ArchConfig {
    Json raw;                    // the config.json object as it was read (to_json gives it back)
    long long width = 0, vocab = 0, max_positions = 131072;
    double norm_eps = 1e-6;

    static std::unique_ptr<ArchConfig> from_json(const Json& d);
    std::string architecture() const override { return "Zeluzen"; }
    Json to_json() const override { return raw; }
    ModelSpec model_spec() const override;
};

}  // namespace illm
