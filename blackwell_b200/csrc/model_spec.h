// What a config.json model consists of: the layer list in the terms of the layered model's mechanisms, filled in by the
// reader of the architecture that config.json names.
#pragma once
#include <string>
#include <vector>

#include "json.h"

namespace bw {

// Rotary positions on the first `dims` dimensions: pair i turns by position * frequency(i).
struct Rotation {
    int dims = 0;
    double base = 1;
    // YaRN: pairs that turn fewer than `slow` times within the `original` context run `factor` times slower, those above
    // `fast` turns keep their frequency, and cos / sin are scaled by gain().  factor 0: no scaling.
    double factor = 0, original = 0, fast = 0, slow = 0;
    double frequency(int i) const;
    double gain() const;
    bool operator<(const Rotation& o) const { return key() < o.key(); }
    bool operator==(const Rotation& o) const { return key() == o.key(); }

private:
    std::vector<double> key() const { return {(double)dims, base, factor, original, fast, slow}; }
};

struct MixerSpec {
    enum Kind { kMamba2, kLatentAttention, kRetention, kDelta, kDiffAttention };
    Kind kind = kMamba2;
    int heads = 0, vdim = 0;
    // mamba2
    int state = 0, groups = 1, norm_groups = 1;
    int conv = 0;              // taps (delta too)
    // attention
    int dim = 0;               // query / key size per head (delta, retention too)
    double scale = 0;
    Rotation rot;
    int kv_from = -1;          // the layer whose cache is read; -1: the layer has its own
    int rot_dim = 0, kv_rank = 0;   // latent attention
    int kv_heads = 0;          // differential attention, delta
    int window = 0;            // keys a position sees, itself included; 0: all
    double diff = 0;           // constant part of the second map's weight
    // retention
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
    double embed_scale = 1;
    // Norms: on every sublayer's output (norm1, norm2), or on its input (norm1, norm2) and its output (norm1b, norm2b).
    bool input_norms = false;
    double norm_offset = 0;        // added to the stored weights of these norms and of the final one
    std::vector<LayerSpec> layers;
};

// Reads <dir>/config.json and dispatches on its "architecture".  Returns false and the reason in `err`.
bool read_model_spec(const std::string& dir, ModelSpec* spec, std::string* err);

}  // namespace bw
