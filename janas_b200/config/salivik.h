// The Salivik decoder's typed configuration (see salivik.cpp).
#pragma once

#include <string>
#include <utility>
#include <vector>

#include "registry.h"

namespace jb {

struct SalivikConfig : ArchConfig {
    struct Rotation {
        long long dims = 0;               // 0: no rotation
        double base = 0;
        bool scaled = false;              // scaling {factor, original, fast, slow}
        double factor = 1, original = 0, fast = 0, slow = 0;
    };
    struct Layer {
        std::string type;                 // "attention", "retention" or "latent_attention"
        long long heads = 0, kv_heads = 0, dim = 0, vdim = 0;
        double scale = 1.0;               // the two attentions
        long long window = 0;             // mask.size; 0: every earlier position is seen
        Rotation rot;
        std::vector<double> decay;        // retention: one number per head
        long long rot_dim = 0, kv_rank = 0, q_rank = 0;      // latent attention
        // feed-forward
        bool has_mlp = false;
        std::string mlp_kind;             // "dense" or "moe"
        long long ff = 0;                 // dense
        double limit = 0;
        long long experts = 0, top = 0, expert_ff = 0, shared_ff = 0;      // moe; shared_ff 0: no shared expert
        double expert_limit = 0, shared_limit = 0;
    };
    long long vocab = 0, width = 0;
    double norm_eps = 0;
    bool has_loop = false;
    long long loop_start = 0, loop_stop = 0, loop_times = 1;
    std::vector<Layer> layers;

    static SalivikConfig from_json(const Json &config_json);
    void validate() const;
    // (layer, whether a pass begins with it) in the order the layers run
    std::vector<std::pair<int, bool>> order() const;

    std::string architecture() const override { return "Salivik"; }
    Json to_json() const override;
    ModelSpec to_model_spec() const override;
};

void register_salivik();

}  // namespace jb
