// Readers of config.json, one per architecture, and the table of the architectures.
#include "model_spec.h"

#include <stdio.h>
#include <string.h>

#include "../../include/blackwell_b200.h"

namespace bw {
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

bool read_latent(const Json& m, const std::string& at, int layer, const ModelSpec& model, Reader& r, MixerSpec* s) {
    s->kind = MixerSpec::kLatentAttention;
    s->dim = r.integer(m, "dim", at, 1);
    s->rot_dim = r.integer(m, "rot_dim", at, 1);
    s->kv_rank = r.integer(m, "kv_rank", at, 1, 2048);
    s->scale = r.real(m, "scale", at);
    const Json* rot = r.need(m, "rot", at);
    if (rot) {
        s->rot_dims = r.integer(*rot, "dims", at + " rot", 0, s->rot_dim);
        s->rot_base = r.real(*rot, "base", at + " rot");
        if (r.ok && (s->rot_dims % 2 != 0 || !(s->rot_base > 0))) r.fail(at + ": bad rotation");
    }
    const Json* from = m.get("kv_from");
    if (from && !from->is_null()) {
        s->kv_from = r.integer(m, "kv_from", at, 0, layer - 1);
        if (!r.ok) return false;
        const MixerSpec& o = model.layers[s->kv_from].mixer;
        if (o.kind != MixerSpec::kLatentAttention || o.kv_from >= 0 || o.kv_rank != s->kv_rank || o.rot_dim != s->rot_dim ||
            o.rot_dims != s->rot_dims || o.rot_base != s->rot_base)
            r.fail(at + ": 'kv_from' names a layer whose cache does not fit");
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
        if (type->str == "mamba2") read_mamba2(*m, at, r, &s.mixer);
        else if (type->str == "latent_attention") read_latent(*m, at, (int)i, *spec, r, &s.mixer);
        else if (type->str == "retention") read_retention(*m, at, r, &s.mixer);
        else r.fail(at + ": unknown type '" + type->str + "'");
        const Json* mlp = l.get("mlp");
        if (r.ok && mlp && !mlp->is_null()) {
            const Json* kind = mlp->get("kind");
            if (!kind || kind->str != "dense") r.fail(at + ": unknown feed-forward kind");
            s.ff = r.integer(*mlp, "ff", at + " mlp", 1);
        }
        spec->layers.push_back(s);
    }
    return r.ok;
}

struct Architecture {
    const char* name;
    bool (*read)(const Json&, ModelSpec*, std::string*);
};
const Architecture kArchitectures[] = {
    {"Vifivik", read_vifivik},
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
        if (l.mixer.kv_from >= 0) ++out->shared_cache_layers;
    }
    return 0;
}
