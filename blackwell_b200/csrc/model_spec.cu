// Readers of config.json, one per architecture, and the table of the architectures.
#include "model_spec.h"

#include <math.h>
#include <stdio.h>
#include <string.h>

#include <algorithm>

#include "../../include/blackwell_b200.h"

namespace bw {

double Rotation::frequency(int i) const {
    const double f = pow(base, -2.0 * i / dims);
    if (factor == 0) return f;
    const double pi = 3.14159265358979323846;
    auto pair_of = [&](double turns) { return dims * log(original / (2 * pi * turns)) / (2 * log(base)); };
    const double lo = std::max(floor(pair_of(fast)), 0.0), hi = std::min(ceil(pair_of(slow)), dims - 1.0);
    const double ramp = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
    return f / factor * ramp + f * (1 - ramp);
}
double Rotation::gain() const { return factor == 0 ? 1.0 : 0.1 * log(factor) + 1.0; }

namespace {

struct Reader {   // typed access with one error message
    std::string* err;
    bool ok = true;
    void fail(const std::string& what) { if (ok) { *err = "config.json: " + what; ok = false; } }
    const Json* need(const Json& j, const char* key, const std::string& where) {
        const Json* v = j.get(key);
        if (!v || v->is_null()) fail(where + " has no '" + key + "'");
        return v && !v->is_null() ? v : nullptr;
    }
    int integer(const Json& j, const char* key, const std::string& where, int lo, int hi = 1 << 30) {
        const Json* v = need(j, key, where);
        if (!v) return lo;
        if (!v->is_int() || v->num < lo || v->num > hi) { fail(where + ": '" + key + "' is out of range"); return lo; }
        return (int)v->num;
    }
    double real(const Json& j, const char* key, const std::string& where) {
        const Json* v = need(j, key, where);
        if (!v) return 0;
        if (v->type != Json::kNumber) fail(where + ": '" + key + "' is not a number");
        return v->num;
    }
};

bool read_mamba2(const Json& m, const std::string& at, Reader& r, MixerSpec* s) {
    s->kind = MixerSpec::kMamba2;
    s->state = r.integer(m, "state", at, 1, 512);
    s->groups = r.integer(m, "groups", at, 1);
    s->conv = r.integer(m, "conv", at, 1, 64);
    s->norm_groups = r.integer(m, "norm_groups", at, 1);
    if (r.ok && s->heads % s->groups != 0) r.fail(at + ": 'groups' does not divide 'heads'");
    if (r.ok && (s->heads * s->vdim) % s->norm_groups != 0) r.fail(at + ": 'norm_groups' does not divide the inner size");
    return r.ok;
}

bool read_retention(const Json& m, const std::string& at, Reader& r, MixerSpec* s) {
    s->kind = MixerSpec::kRetention;
    s->dim = r.integer(m, "dim", at, 1, 512);
    const Json* d = r.need(m, "decay", at);
    if (d)
        for (const Json& v : d->arr) {
            if (v.type != Json::kNumber || v.num < 0 || v.num > 1) r.fail(at + ": 'decay' is not in [0, 1]");
            s->decay.push_back(v.num);
        }
    if (r.ok && (int)s->decay.size() != s->heads) r.fail(at + ": 'decay' needs one value per head");
    return r.ok;
}

// 'rot' of a mixer: dims (even, at most `size`), base and, optionally, YaRN scaling.
void read_rotation(const Json& m, const std::string& at, int size, Reader& r, Rotation* rot) {
    const Json* j = r.need(m, "rot", at);
    if (!j) return;
    rot->dims = r.integer(*j, "dims", at + " rot", 0, size);
    rot->base = r.real(*j, "base", at + " rot");
    if (r.ok && (rot->dims % 2 != 0 || !(rot->base > 0))) r.fail(at + ": bad rotation");
    const Json* s = j->get("scaling");
    if (!r.ok || !s || s->is_null()) return;
    rot->factor = r.real(*s, "factor", at + " rot scaling");
    rot->original = r.real(*s, "original", at + " rot scaling");
    rot->fast = r.real(*s, "fast", at + " rot scaling");
    rot->slow = r.real(*s, "slow", at + " rot scaling");
    if (r.ok && !(rot->factor > 0 && rot->original > 0 && rot->fast > 0 && rot->slow > 0 && rot->base != 1))
        r.fail(at + ": bad rotation scaling");
}

// 'kv_from': an earlier layer of the same kind that has a cache of its own.
bool read_kv_from(const Json& m, const std::string& at, int layer, const ModelSpec& model, Reader& r, MixerSpec* s) {
    const Json* from = m.get("kv_from");
    if (!r.ok || !from || from->is_null()) return false;
    s->kv_from = r.integer(m, "kv_from", at, 0, layer - 1);
    if (!r.ok) return false;
    const MixerSpec& o = model.layers[s->kv_from].mixer;
    if (o.kind != s->kind || o.kv_from >= 0 || o.kv_rank != s->kv_rank || o.rot_dim != s->rot_dim || !(o.rot == s->rot) ||
        (s->kind == MixerSpec::kDiffAttention && (o.kv_heads != s->kv_heads || o.dim != s->dim || o.vdim != s->vdim)))
        r.fail(at + ": 'kv_from' names a layer whose cache does not fit");
    return r.ok;
}

bool read_latent(const Json& m, const std::string& at, int layer, const ModelSpec& model, Reader& r, MixerSpec* s) {
    s->kind = MixerSpec::kLatentAttention;
    s->dim = r.integer(m, "dim", at, 1);
    s->rot_dim = r.integer(m, "rot_dim", at, 1);
    s->kv_rank = r.integer(m, "kv_rank", at, 1, 2048);
    s->scale = r.real(m, "scale", at);
    read_rotation(m, at, s->rot_dim, r, &s->rot);
    read_kv_from(m, at, layer, model, r, s);
    return r.ok;
}

bool read_kv_heads(const Json& m, const std::string& at, Reader& r, MixerSpec* s) {
    s->kv_heads = r.integer(m, "kv_heads", at, 1);
    if (r.ok && s->heads % s->kv_heads != 0) r.fail(at + ": 'kv_heads' does not divide 'heads'");
    return r.ok;
}

bool read_delta(const Json& m, const std::string& at, Reader& r, MixerSpec* s) {
    s->kind = MixerSpec::kDelta;
    s->dim = r.integer(m, "dim", at, 1, 512);
    s->conv = r.integer(m, "conv", at, 1, 64);
    return read_kv_heads(m, at, r, s);
}

bool read_diff_attention(const Json& m, const std::string& at, int layer, const ModelSpec& model, Reader& r, MixerSpec* s) {
    s->kind = MixerSpec::kDiffAttention;
    s->dim = r.integer(m, "dim", at, 1, 4096);
    if (r.ok && s->vdim > 2048) r.fail(at + ": 'vdim' is out of range");
    read_kv_heads(m, at, r, s);
    s->scale = r.real(m, "scale", at);
    s->diff = r.real(m, "diff", at);
    const Json* mask = m.get("mask");
    if (mask && !mask->is_null()) s->window = r.integer(*mask, "size", at + " mask", 1);
    read_rotation(m, at, s->dim, r, &s->rot);
    read_kv_from(m, at, layer, model, r, s);
    return r.ok;
}

// 'mlp' of a layer: dense, or null for none.
void read_mlp(const Json& l, const std::string& at, Reader& r, LayerSpec* s) {
    const Json* mlp = l.get("mlp");
    if (!r.ok || !mlp || mlp->is_null()) return;
    const Json* kind = mlp->get("kind");
    if (!kind || kind->str != "dense") r.fail(at + ": unknown feed-forward kind");
    s->ff = r.integer(*mlp, "ff", at + " mlp", 1);
}

// The list 'layers'; `mixer` reads the mixer of one layer by its type.
template <typename F>
bool read_layers(const Json& j, Reader& r, ModelSpec* spec, F mixer) {
    const Json* layers = r.need(j, "layers", "the model");
    if (!r.ok) return false;
    if (layers->type != Json::kArray || layers->arr.empty()) { r.fail("'layers' is not a list"); return false; }
    for (size_t i = 0; i < layers->arr.size() && r.ok; ++i) {
        const Json& l = layers->arr[i];
        const std::string at = "layer " + std::to_string(i);
        const Json *type = r.need(l, "type", at), *m = r.need(l, "mixer", at);
        if (!r.ok) return false;
        LayerSpec s;
        s.mixer.heads = r.integer(*m, "heads", at, 1);
        s.mixer.vdim = r.integer(*m, "vdim", at, 1);
        if (!r.ok) return false;
        mixer(type->str, *m, at, (int)i, &s.mixer);
        read_mlp(l, at, r, &s);
        spec->layers.push_back(s);
    }
    return r.ok;
}

// Vifivik: norms on the sublayer outputs; mamba2, latent attention and retention mixers in any order; gated feed-forward.
bool read_vifivik(const Json& j, ModelSpec* spec, std::string* err) {
    Reader r{err};
    spec->vocab = r.integer(j, "vocab", "the model", 1);
    spec->width = r.integer(j, "width", "the model", 1);
    if (const Json* n = r.need(j, "norm", "the model")) spec->eps = r.real(*n, "eps", "norm");
    const Json* cap = j.get("logit_softcap");
    if (cap && !cap->is_null()) {
        spec->softcap = r.real(j, "logit_softcap", "the model");
        if (r.ok && spec->softcap < 0) r.fail("'logit_softcap' is negative");
    }
    return read_layers(j, r, spec, [&](const std::string& type, const Json& m, const std::string& at, int i, MixerSpec* s) {
        if (type == "mamba2") read_mamba2(m, at, r, s);
        else if (type == "latent_attention") read_latent(m, at, i, *spec, r, s);
        else if (type == "retention") read_retention(m, at, r, s);
        else r.fail(at + ": unknown type '" + type + "'");
    });
}

// Lanedra: norms around every sublayer; gated delta-rule and windowed differential-attention mixers in any order; gated
// feed-forward or none.
bool read_lanedra(const Json& j, ModelSpec* spec, std::string* err) {
    Reader r{err};
    spec->vocab = r.integer(j, "vocab", "the model", 1);
    spec->width = r.integer(j, "width", "the model", 1);
    if (const Json* n = r.need(j, "norm", "the model")) spec->eps = r.real(*n, "eps", "norm");
    if (const Json* e = r.need(j, "embedding", "the model")) spec->embed_scale = r.real(*e, "scale", "embedding");
    spec->input_norms = true;
    spec->norm_offset = 1;
    return read_layers(j, r, spec, [&](const std::string& type, const Json& m, const std::string& at, int i, MixerSpec* s) {
        if (type == "delta") read_delta(m, at, r, s);
        else if (type == "attention") read_diff_attention(m, at, i, *spec, r, s);
        else r.fail(at + ": unknown type '" + type + "'");
    });
}

struct Architecture {
    const char* name;
    bool (*read)(const Json&, ModelSpec*, std::string*);
};
const Architecture kArchitectures[] = {
    {"Vifivik", read_vifivik},
    {"Lanedra", read_lanedra},
};

}  // namespace

bool read_model_spec(const std::string& dir, ModelSpec* spec, std::string* err) {
    const std::string path = dir + "/config.json";
    FILE* f = fopen(path.c_str(), "rb");
    if (!f) { *err = "cannot open " + path; return false; }
    std::string text;
    char buf[65536];
    size_t n;
    while ((n = fread(buf, 1, sizeof buf, f)) > 0) text.append(buf, n);
    fclose(f);
    Json j;
    if (!Json::parse(text.data(), text.size(), &j, err)) { *err = path + ": " + *err; return false; }
    const Json* a = j.get("architecture");
    if (!a || a->type != Json::kString) { *err = path + " names no architecture"; return false; }
    for (const Architecture& k : kArchitectures)
        if (a->str == k.name) {
            spec->architecture = a->str;
            return k.read(j, spec, err);
        }
    *err = path + ": architecture '" + a->str + "' is not known";
    return false;
}

}  // namespace bw

extern "C" int bw_model_probe(const char* dir, bw_model_info* out, char* message, int message_bytes) {
    if (!dir || !out) return cudaErrorInvalidValue;
    bw::ModelSpec spec;
    std::string err;
    const bool ok = bw::read_model_spec(dir, &spec, &err);
    if (message && message_bytes > 0) snprintf(message, (size_t)message_bytes, "%s", err.c_str());
    if (!ok) return cudaErrorInvalidValue;
    memset(out, 0, sizeof *out);
    snprintf(out->architecture, sizeof out->architecture, "%s", spec.architecture.c_str());
    out->layers = (int)spec.layers.size();
    out->width = spec.width;
    out->vocab = spec.vocab;
    for (const bw::LayerSpec& l : spec.layers) {
        if (l.mixer.kind == bw::MixerSpec::kMamba2) ++out->mamba2_layers;
        if (l.mixer.kind == bw::MixerSpec::kRetention) ++out->retention_layers;
        if (l.mixer.kind == bw::MixerSpec::kLatentAttention) ++out->latent_layers;
        if (l.mixer.kind == bw::MixerSpec::kDelta) ++out->delta_layers;
        if (l.mixer.kind == bw::MixerSpec::kDiffAttention) ++out->diff_attention_layers;
        if (l.mixer.kv_from >= 0) ++out->shared_cache_layers;
    }
    return 0;
}
