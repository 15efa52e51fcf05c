// The Dafalix decoder's typed configuration (see dafalix.cpp).
#pragma once

#include <string>
#include <vector>

#include "registry.h"

namespace jb {

struct DafalixConfig : ArchConfig {
    struct Layer {
        std::string type;                 // "parallel" or "mlstm"
        // "mlstm", and the attention side of "parallel"
        long long heads = 0, kv_heads = 0, dim = 0, vdim = 0;
        double gate_cap = 0;              // mlstm
        double scale = 1.0;               // attention
        long long window = 0;             // mask.size; 0: every earlier position is seen
        long long rot_dims = 0;           // 0: no rotation
        double rot_base = 0, rot_factor = 1.0;
        bool rot_scaled = false;          // rot.scaling stands in the file
        // the recurrent side of "parallel"
        long long rec_width = 0, rec_blocks = 1, rec_conv = 1;
        double left_scale = 1.0, right_scale = 1.0;
        // feed-forward
        bool has_mlp = false;
        long long experts = 0, top = 0, expert_ff = 0;
    };
    long long vocab = 0, width = 0, streams = 1;
    double norm_eps = 0, residual_mult = 1.0;
    bool has_loop = false;
    long long loop_start = 0, loop_stop = 0, loop_times = 1;
    std::vector<Layer> layers;

    static DafalixConfig from_json(const Json &config_json);
    void validate() const;
    std::vector<int> order() const;       // the layers in the order they run

    std::string architecture() const override { return "Dafalix"; }
    Json to_json() const override;
    ModelSpec to_model_spec() const override;
};

void register_dafalix();

}  // namespace jb
