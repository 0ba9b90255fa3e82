// What a config.json model consists of: the layer list in the terms of the layered model's mechanisms, filled in by the
// reader of the architecture that config.json names.
#pragma once
#include <string>
#include <vector>

#include "json.h"

namespace bw {

struct MixerSpec {
    enum Kind { kMamba2, kLatentAttention, kRetention };
    Kind kind = kMamba2;
    int heads = 0, vdim = 0;
    // mamba2
    int state = 0, groups = 1, conv = 0, norm_groups = 1;
    // latent attention
    int dim = 0, rot_dim = 0, kv_rank = 0, rot_dims = 0;
    int kv_from = -1;          // the layer whose cache is read; -1: the layer has its own
    double rot_base = 0, scale = 0;
    // retention (dim above)
    std::vector<double> decay;
};
struct LayerSpec {
    MixerSpec mixer;
    int ff = 0;                // 0: no feed-forward
};
struct ModelSpec {
    std::string architecture;
    int vocab = 0, width = 0;
    double eps = 0, softcap = 0;   // softcap 0: none
    std::vector<LayerSpec> layers;
};

// Reads <dir>/config.json and dispatches on its "architecture".  Returns false and the reason in `err`.
bool read_model_spec(const std::string& dir, ModelSpec* spec, std::string* err);

}  // namespace bw
