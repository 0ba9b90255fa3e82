// Models described by a config.json (model_spec.h): a list of layers, each a mixer and an optional feed-forward, with norms
// on the sublayers' outputs -- x <- x + norm1(mixer(x)), x <- x + norm2(ff(x)) -- or on both sides -- x <- x +
// norm1b(mixer(norm1(x))), x <- x + norm2b(ff(norm2(x))) --, an fp32 residual stream, and logits = softcap(head norm(x)).
// Mixers: mamba2, retention, gated delta rule (all on the gated linear recurrence), latent attention, differential attention.
//
// Weights are bfloat16 and stay so on the device; matrices that read the same input are stacked by rows, gate and up
// rows are interleaved (the product's epilogue applies silu(gate) * up), head blocks are padded to multiples of eight
// with zero rows / columns.  Two activation formats: bfloat16 (serving) and fp32 (cfg.compute_f32).
//
// Per-slot state: for every attention layer that owns a cache, in the activation format, [slot][max_seq][latent | rotated key
// part] (latent) or a ring [slot][cap][key / value heads] that holds the longest window of the layers that read it and one
// portion (differential); for every recurrent layer the fp32 state and, for mamba2 and delta, the last inputs of the
// convolution.  A slot needs no clearing when it is used again: at position 0 states and convolution inputs count as zero,
// and attention reads positions below the current one only.
#include <cuda_runtime.h>
#include <math.h>

#include <algorithm>
#include <map>

#include "decode_model.h"
#include "host_util.h"
#include "lm_ops.h"
#include "model_spec.h"
#include "safetensors.h"

namespace bw {
namespace {

using lm::bf16;
using lm::pad8;

constexpr int kAbsorbedRows = 16;   // portions up to this many rows attend in the latent space like decode steps
constexpr int kLogitRows = 64;      // rows of logits per head product of a portion

struct Mat {   // device matrix [N][ld]
    bf16* p = nullptr;
    int N = 0, K = 0, ld = 0;
};

// Host image of a matrix under construction.
struct Stack {
    int K, ld, rows = 0;
    std::vector<uint16_t> data;
    explicit Stack(int k) : K(k), ld(pad8(k)) {}
    uint16_t* row(int r) { return &data[(size_t)r * ld]; }
    void grow(int n) { rows += n; data.resize((size_t)rows * ld, 0); }
    // rows of `src` [n][K] in blocks of `per` rows, each padded to pad8(per)
    void add(const std::vector<uint16_t>& src, int n, int per, int padded) {
        const int base = rows;
        grow(n / per * padded);
        for (int i = 0; i < n; ++i) std::copy_n(&src[(size_t)i * K], K, row(base + i / per * padded + i % per));
    }
    void add(const std::vector<uint16_t>& src, int n) { add(src, n, n, n); }
};

struct Loader {
    SafeTensors st;
    DecodeContext& ctx;
    explicit Loader(DecodeContext& c) : ctx(c) {}
    int bad() { return -3; }
    int tensor(const std::string& name, const std::vector<long>& shape, std::vector<uint16_t>* out) {
        return st.read_bf16(name, shape, out, &ctx.error) ? 0 : bad();
    }
    int floats(const std::string& name, const std::vector<long>& shape, std::vector<float>* f) {   // appended
        std::vector<uint16_t> h;
        BW_TRY(tensor(name, shape, &h));
        for (uint16_t v : h) {
            const uint32_t u = (uint32_t)v << 16;
            float x;
            memcpy(&x, &u, 4);
            f->push_back(x);
        }
        return 0;
    }
    int vec(const std::string& name, const std::vector<long>& shape, float** dev, double offset = 0) {   // fp32 on the device
        std::vector<float> f;
        BW_TRY(floats(name, shape, &f));
        if (offset != 0)
            for (float& x : f) x = (float)(x + offset);
        return ctx.upload(dev, f);
    }
    int upload(const Stack& s, Mat* m) {
        m->N = s.rows;
        m->K = s.K;
        m->ld = s.ld;
        uint16_t* p = nullptr;
        BW_TRY(ctx.upload(&p, s.data));
        m->p = reinterpret_cast<bf16*>(p);
        return 0;
    }
    int matrix(const std::string& name, int N, int K, Mat* m) {
        std::vector<uint16_t> h;
        BW_TRY(tensor(name, {N, K}, &h));
        Stack s(K);
        s.add(h, N);
        return upload(s, m);
    }
    // [N][heads * V] with every head's columns padded to pad8(V)
    int matrix_by_heads(const std::string& name, int N, int heads, int V, Mat* m) {
        std::vector<uint16_t> h;
        BW_TRY(tensor(name, {N, (long)heads * V}, &h));
        Stack s(heads * pad8(V));
        s.grow(N);
        for (int n = 0; n < N; ++n)
            for (int i = 0; i < heads; ++i) std::copy_n(&h[((size_t)n * heads + i) * V], V, s.row(n) + i * pad8(V));
        return upload(s, m);
    }
};

// Work buffers shared by all layers: largest need over the layers, in elements per row unless noted.
struct Work {
    long proj = 0, proj32 = 0, conv = 0, mixed = 0, ff = 0, o32 = 0, heads = 0;   // per row
    long absorbed_bytes = 0, part = 0, kv = 0, chunk_bytes = 0;                   // whole buffers
    void *xb = nullptr, *proj_b = nullptr, *conv_b = nullptr, *mixed_b = nullptr, *ff_b = nullptr, *fin_b = nullptr;
    float *proj32_b = nullptr, *o32_b = nullptr, *log_decay = nullptr, *weight = nullptr, *sub = nullptr, *part_b = nullptr;
    void *qabs_b = nullptr, *kv_b = nullptr, *chunk_b = nullptr;
    long ldx = 0;
};

struct Env {   // fixed properties of an engine
    int f32 = 0, slots = 0, max_seq = 0, max_rows = 0, width = 0, sms = 148;
    float eps = 0;
    int elem() const { return f32 ? 4 : 2; }
    char* at(void* base, long elems) const { return static_cast<char*>(base) + elems * elem(); }
};

int project(const Env& e, const Work& w, const Mat& m, const void* x, long ldx, int T, void* y, long ldy, float* y32, long ldy32,
            int split, cudaStream_t st) {
    lm::LinearArgs a{};
    a.x = x; a.ldx = ldx; a.W = m.p; a.ldw = m.ld; a.T = T; a.N = m.N; a.K = m.K;
    a.y = y; a.ldy = ldy; a.y32 = y32; a.ldy32 = ldy32; a.split = split; a.f32 = e.f32;
    return lm::linear(a, st);
}

class Mixer {
public:
    explicit Mixer(const MixerSpec& s) : s_(s) {}
    virtual ~Mixer() {}
    virtual int load(Loader& l, const std::string& p, int width) = 0;
    virtual int alloc(DecodeContext& ctx, const Env& e, Work* w) = 0;   // per-slot state; raises the work sizes
    virtual int run(const Env& e, const Work& w, const lm::Rows& r, cudaStream_t st) = 0;   // w.xb -> w.mixed_b
    int mixed_ld() const { return s_.heads * pad8(s_.vdim); }
    const Mat& out() const { return o_; }
    const MixerSpec& spec() const { return s_; }
    virtual bool rotates() const { return false; }   // takes cos / sin of spec().rot
    void set_rotation(const float2* cs) { cs_ = cs; }

protected:
    MixerSpec s_;
    Mat in_, o_;
    const float2* cs_ = nullptr;
};

// Recurrent mixers: N x vdim state per head, gated norm on the read-out.
class RecurrentMixer : public Mixer {
public:
    using Mixer::Mixer;

protected:
    int N_ = 0;
    float* S_ = nullptr;
    int alloc_recurrent(DecodeContext& ctx, const Env& e, Work* w) {
        const long inner = mixed_ld();
        w->mixed = std::max(w->mixed, inner);
        w->o32 = std::max(w->o32, inner);
        return ctx.alloc(&S_, (size_t)e.slots * s_.heads * N_ * pad8(s_.vdim));
    }
    lm::RecurrenceArgs recurrence(const Work& w) const {
        lm::RecurrenceArgs a{};
        a.heads = s_.heads; a.N = N_; a.V = s_.vdim; a.S = S_; a.o = w.o32_b; a.ldo = mixed_ld();
        return a;
    }
    // chunks on the tensor cores from 16 rows on (bf16); token by token with fp32 FMAs otherwise
    int recur(const Env& e, const lm::RecurrenceArgs& a, const lm::Rows& r, cudaStream_t st) const {
        if (!e.f32 && !r.row_slot && r.T >= 16) {
            if (a.delta && lm::delta_chunk_supported(a)) return lm::delta_chunk(a, r, st);
            if (!a.delta && lm::recurrence_chunk_supported(a)) return lm::recurrence_chunk(a, r, st);
        }
        return lm::recurrence_step(a, nullptr, r, e.f32, st);
    }
};

class Mamba2 : public RecurrentMixer {
public:
    explicit Mamba2(const MixerSpec& s) : RecurrentMixer(s) { N_ = s.state; }
    int load(Loader& l, const std::string& p, int width) override {
        const int inner = s_.heads * s_.vdim, gn = s_.groups * s_.state, channels = inner + 2 * gn;
        std::vector<uint16_t> h;
        BW_TRY(l.tensor(p + "in", {2L * inner + 2 * gn + s_.heads, width}, &h));
        Stack st(width);
        auto part = [&](int first, int n) { return std::vector<uint16_t>(h.begin() + (size_t)first * width, h.begin() + (size_t)(first + n) * width); };
        st.add(part(0, inner), inner, s_.vdim, pad8(s_.vdim));                       // z
        st.add(part(inner, inner), inner, s_.vdim, pad8(s_.vdim));                   // x
        st.add(part(2 * inner, 2 * gn), 2 * gn, s_.state, pad8(s_.state));           // B, C
        split_ = st.rows;
        st.add(part(2 * inner + 2 * gn, s_.heads), s_.heads);                        // dt
        BW_TRY(l.upload(st, &in_));
        BW_TRY(l.vec(p + "conv", {channels, s_.conv}, &conv_w_));
        BW_TRY(l.vec(p + "conv.b", {channels}, &conv_b_));
        BW_TRY(l.vec(p + "dt_bias", {s_.heads}, &dt_bias_));
        BW_TRY(l.vec(p + "A_log", {s_.heads}, &A_log_));
        BW_TRY(l.vec(p + "D", {s_.heads}, &D_));
        BW_TRY(l.vec(p + "norm", {inner}, &norm_));
        return l.matrix_by_heads(p + "o", width, s_.heads, s_.vdim, &o_);
    }
    int alloc(DecodeContext& ctx, const Env& e, Work* w) override {
        w->proj = std::max(w->proj, (long)split_);
        w->proj32 = std::max(w->proj32, (long)s_.heads);
        w->conv = std::max(w->conv, (long)split_ - mixed_ld());
        w->heads = std::max(w->heads, (long)s_.heads);
        BW_TRY(ctx.alloc(&ring_, (size_t)e.slots * s_.conv * (s_.heads * s_.vdim + 2 * s_.groups * s_.state)));
        return alloc_recurrent(ctx, e, w);
    }
    int run(const Env& e, const Work& w, const lm::Rows& r, cudaStream_t st) override {
        const int inner8 = mixed_ld(), bc = s_.groups * pad8(s_.state);
        BW_TRY(project(e, w, in_, w.xb, w.ldx, r.T, w.proj_b, split_, w.proj32_b, s_.heads, split_, st));
        lm::ConvArgs c{};
        c.u = w.proj_b; c.ldu = split_; c.w = conv_w_; c.bias = conv_b_; c.ring = ring_; c.taps = s_.conv; c.heads = s_.heads;
        c.V = s_.vdim; c.N = s_.state; c.groups = s_.groups; c.off = inner8; c.out = w.conv_b; c.ldo = split_ - inner8;
        c.dt_raw = w.proj32_b; c.ld_dt = s_.heads; c.dt_bias = dt_bias_; c.A_log = A_log_; c.log_decay = w.log_decay; c.weight = w.weight;
        lm::RecurrenceArgs a = recurrence(w);
        a.groups = s_.groups; a.D = D_;
        if (r.row_slot) {
            BW_TRY(lm::recurrence_step(a, &c, r, e.f32, st));
        } else {
            BW_TRY(lm::conv_silu(c, r, e.f32, st));
            BW_TRY(lm::conv_ring_store(c, r, e.f32, st));
            a.v = w.conv_b; a.k = e.at(w.conv_b, inner8); a.q = e.at(w.conv_b, inner8 + bc);
            a.ldq = a.ldk = a.ldv = c.ldo;
            a.log_decay = w.log_decay; a.weight = w.weight;
            BW_TRY(recur(e, a, r, st));
        }
        return lm::gated_norm(w.mixed_b, inner8, w.o32_b, inner8, w.proj_b, split_, norm_, r.T, s_.heads, s_.vdim, s_.norm_groups, 1, e.eps,
                              e.f32, st);
    }

private:
    int split_ = 0;
    float *conv_w_ = nullptr, *conv_b_ = nullptr, *dt_bias_ = nullptr, *A_log_ = nullptr, *D_ = nullptr, *norm_ = nullptr, *ring_ = nullptr;
};

class Retention : public RecurrentMixer {
public:
    explicit Retention(const MixerSpec& s) : RecurrentMixer(s) { N_ = s.dim; }
    int load(Loader& l, const std::string& p, int width) override {
        const int H = s_.heads, qk = H * s_.dim, v = H * s_.vdim;
        std::vector<uint16_t> h;
        Stack st(width);
        for (const char* name : {"q", "k"}) {
            BW_TRY(l.tensor(p + name, {qk, width}, &h));
            st.add(h, qk, s_.dim, pad8(s_.dim));
        }
        for (const char* name : {"v", "g"}) {
            BW_TRY(l.tensor(p + name, {v, width}, &h));
            st.add(h, v, s_.vdim, pad8(s_.vdim));
        }
        BW_TRY(l.upload(st, &in_));
        std::vector<float> ld(H);
        for (int i = 0; i < H; ++i) ld[i] = s_.decay[i] > 0 ? (float)std::max(log(s_.decay[i]), -1e4) : -1e4f;
        BW_TRY(l.ctx.upload(&log_decay_, ld));
        return l.matrix_by_heads(p + "o", width, H, s_.vdim, &o_);
    }
    int alloc(DecodeContext& ctx, const Env& e, Work* w) override {
        w->proj = std::max(w->proj, (long)in_.N);
        return alloc_recurrent(ctx, e, w);
    }
    int run(const Env& e, const Work& w, const lm::Rows& r, cudaStream_t st) override {
        const int qk8 = s_.heads * pad8(s_.dim), v8 = mixed_ld();
        BW_TRY(project(e, w, in_, w.xb, w.ldx, r.T, w.proj_b, in_.N, nullptr, 0, in_.N, st));
        lm::RecurrenceArgs a = recurrence(w);
        a.groups = s_.heads;
        a.q = w.proj_b; a.k = e.at(w.proj_b, qk8); a.v = e.at(w.proj_b, 2L * qk8);
        a.ldq = a.ldk = a.ldv = in_.N;
        a.head_log_decay = log_decay_;
        a.const_weight = (float)(1.0 / sqrt((double)s_.dim));
        BW_TRY(recur(e, a, r, st));
        return lm::gated_norm(w.mixed_b, v8, w.o32_b, v8, e.at(w.proj_b, 2L * qk8 + v8), in_.N, nullptr, r.T, s_.heads, s_.vdim, s_.heads, 0,
                              e.eps, e.f32, st);
    }

private:
    float* log_decay_ = nullptr;
};

class GatedDelta : public RecurrentMixer {
public:
    explicit GatedDelta(const MixerSpec& s) : RecurrentMixer(s) { N_ = s.dim; }
    int load(Loader& l, const std::string& p, int width) override {
        const int H = s_.heads, qk = s_.kv_heads * s_.dim, v = H * s_.vdim;
        std::vector<uint16_t> h;
        std::vector<float> taps, norm;
        Stack st(width);
        BW_TRY(l.tensor(p + "g", {v, width}, &h));
        st.add(h, v, s_.vdim, pad8(s_.vdim));
        for (const char* name : {"v", "k", "q"}) {
            const bool values = name[0] == 'v';
            const int n = values ? v : qk, per = values ? s_.vdim : s_.dim;
            BW_TRY(l.tensor(p + name, {n, width}, &h));
            st.add(h, n, per, pad8(per));
            BW_TRY(l.floats(p + name + ".conv", {n, s_.conv}, &taps));
        }
        split_ = st.rows;
        for (const char* name : {"a", "b"}) {
            BW_TRY(l.tensor(p + name, {H, width}, &h));
            st.add(h, H);
        }
        BW_TRY(l.upload(st, &in_));
        BW_TRY(l.ctx.upload(&conv_w_, taps));
        BW_TRY(l.vec(p + "dt_bias", {H}, &dt_bias_));
        BW_TRY(l.vec(p + "A_log", {H}, &A_log_));
        for (int i = 0; i < H; ++i) BW_TRY(l.floats(p + "norm", {s_.vdim}, &norm));   // shared by the heads
        BW_TRY(l.ctx.upload(&norm_, norm));
        return l.matrix_by_heads(p + "o", width, H, s_.vdim, &o_);
    }
    int alloc(DecodeContext& ctx, const Env& e, Work* w) override {
        w->proj = std::max(w->proj, (long)split_);
        w->proj32 = std::max(w->proj32, 2L * s_.heads);
        w->conv = std::max(w->conv, (long)split_ - mixed_ld());
        w->heads = std::max(w->heads, (long)s_.heads);
        if (!e.f32) w->chunk_bytes = std::max(w->chunk_bytes, (long)lm::delta_chunk_bytes(e.max_rows, s_.heads));
        BW_TRY(ctx.alloc(&ring_, (size_t)e.slots * s_.conv * (s_.heads * s_.vdim + 2 * s_.kv_heads * s_.dim)));
        return alloc_recurrent(ctx, e, w);
    }
    int run(const Env& e, const Work& w, const lm::Rows& r, cudaStream_t st) override {
        const int H = s_.heads, inner8 = mixed_ld(), qk8 = s_.kv_heads * pad8(s_.dim);
        BW_TRY(project(e, w, in_, w.xb, w.ldx, r.T, w.proj_b, split_, w.proj32_b, 2 * H, split_, st));
        lm::ConvArgs c{};
        c.u = w.proj_b; c.ldu = split_; c.w = conv_w_; c.ring = ring_; c.taps = s_.conv; c.heads = H; c.V = s_.vdim; c.N = s_.dim;
        c.groups = s_.kv_heads; c.off = inner8; c.out = w.conv_b; c.ldo = split_ - inner8; c.dt_raw = w.proj32_b; c.ld_dt = 2 * H;
        c.beta_raw = w.proj32_b + H; c.dt_bias = dt_bias_; c.A_log = A_log_; c.log_decay = w.log_decay; c.weight = w.weight;
        lm::RecurrenceArgs a = recurrence(w);
        a.groups = s_.kv_heads; a.delta = 1; a.unit_eps = 1e-6f; a.q_scale = (float)(1.0 / sqrt((double)s_.dim)); a.chunk_scratch = w.chunk_b;
        if (r.row_slot) {
            BW_TRY(lm::recurrence_step(a, &c, r, e.f32, st));
        } else {
            BW_TRY(lm::conv_silu(c, r, e.f32, st));
            BW_TRY(lm::conv_ring_store(c, r, e.f32, st));
            a.v = w.conv_b; a.k = e.at(w.conv_b, inner8); a.q = e.at(w.conv_b, inner8 + qk8);
            a.ldq = a.ldk = a.ldv = c.ldo;
            a.log_decay = w.log_decay; a.weight = w.weight;
            BW_TRY(recur(e, a, r, st));
        }
        return lm::gated_norm(w.mixed_b, inner8, w.o32_b, inner8, w.proj_b, split_, norm_, r.T, H, s_.vdim, H, 0, e.eps, e.f32, st);
    }

private:
    int split_ = 0;
    float *conv_w_ = nullptr, *dt_bias_ = nullptr, *A_log_ = nullptr, *norm_ = nullptr, *ring_ = nullptr;
};

class DiffAttention : public Mixer {
public:
    DiffAttention(const MixerSpec& s, DiffAttention* owner) : Mixer(s), owner_(owner), reach_(s.window) {
        if (owner && (reach_ == 0 || (owner->reach_ > 0 && reach_ > owner->reach_))) owner->reach_ = reach_;
    }
    int load(Loader& l, const std::string& p, int width) override {
        const int H = s_.heads, G = s_.kv_heads;
        std::vector<uint16_t> h;
        Stack st(width);
        BW_TRY(l.tensor(p + "q", {2L * H * s_.dim, width}, &h));
        st.add(h, 2 * H * s_.dim, s_.dim, pad8(s_.dim));
        if (!owner_) {
            k_ = st.rows;
            BW_TRY(l.tensor(p + "k", {2L * G * s_.dim, width}, &h));
            st.add(h, 2 * G * s_.dim, s_.dim, pad8(s_.dim));
            v_ = st.rows;
            BW_TRY(l.tensor(p + "v", {(long)G * s_.vdim, width}, &h));
            st.add(h, G * s_.vdim, s_.vdim, pad8(s_.vdim));
        }
        BW_TRY(l.upload(st, &in_));
        double dot[2] = {};
        const char* pairs[2][2] = {{"lq1", "lk1"}, {"lq2", "lk2"}};
        for (int i = 0; i < 2; ++i) {
            std::vector<float> a, b;
            BW_TRY(l.floats(p + pairs[i][0], {s_.dim}, &a));
            BW_TRY(l.floats(p + pairs[i][1], {s_.dim}, &b));
            for (int d = 0; d < s_.dim; ++d) dot[i] += (double)a[d] * b[d];
        }
        lambda_ = (float)(exp(dot[0]) - exp(dot[1]) + s_.diff);
        return l.matrix_by_heads(p + "o", width, H, s_.vdim, &o_);
    }
    int alloc(DecodeContext& ctx, const Env& e, Work* w) override {
        if (!lm::diff_attention_supported(base(e))) { ctx.error = "differential attention: these sizes are not supported"; return cudaErrorInvalidValue; }
        w->proj = std::max(w->proj, (long)in_.N);
        w->mixed = std::max(w->mixed, (long)mixed_ld());
        if (owner_) return 0;
        cap_ = reach_ > 0 ? (int)std::min<long>(e.max_seq, ((long)reach_ - 1 + e.max_rows + 15) / 16 * 16) : e.max_seq;
        char* c = nullptr;
        BW_TRY(ctx.alloc(&c, (size_t)e.slots * cap_ * s_.kv_heads * lm::diff_row(s_.dim, s_.vdim) * e.elem()));
        cache_ = c;
        return 0;
    }
    int run(const Env& e, const Work& w, const lm::Rows& r, cudaStream_t st) override {
        BW_TRY(project(e, w, in_, w.xb, w.ldx, r.T, w.proj_b, in_.N, nullptr, 0, in_.N, st));
        lm::DiffAttnArgs a = base(e);
        const DiffAttention* own = owner_ ? owner_ : this;
        a.cache = own->cache_; a.cap = own->cap_; a.slots = e.slots;
        a.q = w.proj_b; a.ld = in_.N;
        if (!owner_) {
            a.k = e.at(w.proj_b, k_);
            a.v = e.at(w.proj_b, v_);
        }
        a.out = w.mixed_b; a.ldout = mixed_ld();
        a.splits = lm::diff_attention_splits(a, r.T, e.f32);
        return lm::diff_attention(a, r, e.f32, st);
    }
    bool rotates() const override { return true; }

private:
    lm::DiffAttnArgs base(const Env& e) const {
        lm::DiffAttnArgs a{};
        a.heads = s_.heads; a.kv_heads = s_.kv_heads; a.dim = s_.dim; a.V = s_.vdim; a.window = s_.window; a.rot_dims = s_.rot.dims; a.cs = cs_;
        a.max_seq = e.max_seq; a.scale = (float)s_.scale; a.lambda = lambda_; a.out_scale = (float)(1.0 - s_.diff); a.eps = e.eps;
        return a;
    }
    DiffAttention* owner_;
    int reach_;                // longest window over this layer's cache, 0: everything
    int k_ = 0, v_ = 0;        // columns of the projection
    int cap_ = 0;
    float lambda_ = 0;
    void* cache_ = nullptr;
};

class LatentAttention : public Mixer {
public:
    LatentAttention(const MixerSpec& s, LatentAttention* owner) : Mixer(s), owner_(owner) {}
    int load(Loader& l, const std::string& p, int width) override {
        const int H = s_.heads, q = s_.dim + s_.rot_dim;
        std::vector<uint16_t> h;
        Stack st(width);
        BW_TRY(l.tensor(p + "q", {(long)H * q, width}, &h));
        st.grow(H * q8());
        for (int i = 0; i < H; ++i)
            for (int d = 0; d < q; ++d)
                std::copy_n(&h[((size_t)i * q + d) * width], width, st.row(i * q8() + (d < s_.dim ? d : pad8(s_.dim) + d - s_.dim)));
        split_ = st.rows;
        if (!owner_) {
            BW_TRY(l.tensor(p + "dkv", {s_.kv_rank + s_.rot_dim, width}, &h));
            st.add(h, s_.kv_rank + s_.rot_dim);
            BW_TRY(l.vec(p + "dkv.norm", {s_.kv_rank}, &dkv_norm_));
        }
        BW_TRY(l.tensor(p + "g", {H, width}, &h));
        st.add(h, H);
        BW_TRY(l.upload(st, &in_));
        Stack kv(s_.kv_rank);
        BW_TRY(l.tensor(p + "uk", {(long)H * s_.dim, s_.kv_rank}, &h));
        kv.add(h, H * s_.dim, s_.dim, pad8(s_.dim));
        BW_TRY(l.tensor(p + "uv", {(long)H * s_.vdim, s_.kv_rank}, &h));
        kv.add(h, H * s_.vdim, s_.vdim, pad8(s_.vdim));
        BW_TRY(l.upload(kv, &kv_));
        BW_TRY(l.vec(p + "sink", {H}, &sink_));
        return l.matrix_by_heads(p + "o", width, H, s_.vdim, &o_);
    }
    int alloc(DecodeContext& ctx, const Env& e, Work* w) override {
        lm::LatentArgs a = base(e);
        if (!lm::latent_absorbed_supported(a)) { ctx.error = "latent attention: these sizes are not supported"; return cudaErrorInvalidValue; }
        expanded_ = !e.f32 && lm::latent_expanded_supported(a);
        const int rows = expanded_ ? std::max(e.slots, kAbsorbedRows) : std::max(e.slots, e.max_rows);
        w->proj = std::max(w->proj, (long)split_);
        w->proj32 = std::max(w->proj32, (long)in_.N - split_);
        w->mixed = std::max(w->mixed, (long)mixed_ld());
        w->absorbed_bytes = std::max(w->absorbed_bytes, 4L * rows * s_.heads * lm::latent_dp(s_.kv_rank, s_.rot_dim));
        for (int T = 1; T <= rows; ++T) w->part = std::max(w->part, (long)T * s_.heads * splits(e, T) * (pad8(s_.kv_rank) + lm::kPartStats));
        if (expanded_) w->kv = std::max(w->kv, (long)e.max_seq * s_.heads * (pad8(s_.dim) + pad8(s_.vdim)));
        if (owner_) return 0;
        char* c = nullptr;
        BW_TRY(ctx.alloc(&c, (size_t)e.slots * e.max_seq * lm::latent_row(s_.kv_rank, s_.rot_dim) * e.elem()));
        cache_ = c;
        return 0;
    }
    int run(const Env& e, const Work& w, const lm::Rows& r, cudaStream_t st) override {
        const int ld32 = in_.N - split_;
        BW_TRY(project(e, w, in_, w.xb, w.ldx, r.T, w.proj_b, split_, w.proj32_b, ld32, split_, st));
        lm::LatentArgs a = base(e);
        a.q = w.proj_b; a.ldq = split_; a.ld32 = ld32;
        a.dkv = owner_ ? nullptr : w.proj32_b;
        a.gate = w.proj32_b + (owner_ ? 0 : s_.kv_rank + s_.rot_dim);
        a.dkv_norm = dkv_norm_; a.Wkv = kv_.p; a.ldw = kv_.ld; a.sink = sink_; a.out = w.mixed_b; a.ldout = mixed_ld();
        a.cache = owner_ ? owner_->cache_ : cache_;
        a.qabs = w.qabs_b; a.part = w.part_b; a.kv = w.kv_b; a.splits = splits(e, r.T);
        if (expanded_ && !r.row_slot && r.T > kAbsorbedRows) return lm::latent_expanded(a, r, st);
        return lm::latent_absorbed(a, r, e.f32, st);
    }
    bool rotates() const override { return true; }

private:
    int q8() const { return pad8(s_.dim) + pad8(s_.rot_dim); }
    // context splits of an absorbed call with T rows: one CTA per SM, at least one 64-key tile each at full length
    int splits(const Env& e, int T) const {
        const int blocks = T * (e.f32 ? s_.heads : (s_.heads + 15) / 16);
        return std::max(1, std::min({64, (e.max_seq + 63) / 64, e.sms / blocks}));
    }
    lm::LatentArgs base(const Env& e) const {
        lm::LatentArgs a{};
        a.heads = s_.heads; a.dim = s_.dim; a.rot = s_.rot_dim; a.V = s_.vdim; a.R = s_.kv_rank; a.rot_dims = s_.rot.dims;
        a.scale = (float)s_.scale; a.eps = e.eps; a.cs = cs_; a.max_seq = e.max_seq; a.ldc = lm::latent_row(s_.kv_rank, s_.rot_dim);
        return a;
    }
    LatentAttention* owner_;
    bool expanded_ = false;
    int split_ = 0;
    Mat kv_;
    float *dkv_norm_ = nullptr, *sink_ = nullptr;
    void* cache_ = nullptr;
};

struct Layer {
    std::unique_ptr<Mixer> mixer;
    float *in1 = nullptr, *in2 = nullptr;     // norms of the sublayers' inputs, NULL: none
    float *out1 = nullptr, *out2 = nullptr;   // norms of the sublayers' outputs
    Mat gu, down;
    int ff = 0;
};

class LayeredModel : public DecodeModel {
public:
    int load(DecodeContext& ctx, const std::string& dir) override;
    int alloc_state(DecodeContext& ctx) override;
    int enqueue_tokens(DecodeContext& ctx, int rows, const int* slots, const int* pos, const int* tokens, float* logits,
                       cudaStream_t st) override {
        lm::Rows r{};
        r.T = rows; r.row_slot = slots; r.row_pos = pos;
        BW_TRY(enqueue_layers(ctx, r, tokens, st));
        return head(rows, nullptr, logits, st);
    }
    int max_portion() const override { return env_.max_rows; }
    int enqueue_portion(DecodeContext& ctx, int slot, int pos0, int n, const int* tokens, int n_want, const int* want, float* logits,
                        cudaStream_t st) override {
        if (n > 0) {
            lm::Rows r{};
            r.T = n; r.slot = slot; r.pos0 = pos0;
            BW_TRY(enqueue_layers(ctx, r, tokens, st));
        }
        for (int i = 0; i < n_want; i += kLogitRows)
            BW_TRY(head(std::min(kLogitRows, n_want - i), want + i, logits + (size_t)i * spec_.vocab, st));
        return 0;
    }

private:
    int enqueue_layers(DecodeContext& ctx, const lm::Rows& r, const int* tokens, cudaStream_t st);
    int head(int rows, const int* want, float* logits, cudaStream_t st) {
        BW_TRY(lm::norm_rows(w_.fin_b, w_.ldx, x_, final_norm_, want, rows, env_.width, env_.eps, env_.f32, st));
        lm::LinearArgs a{};
        a.x = w_.fin_b; a.ldx = w_.ldx; a.W = head_.p; a.ldw = head_.ld; a.T = rows; a.N = head_.N; a.K = head_.K;
        a.y = logits; a.ldy = head_.N; a.y_f32 = 1; a.split = head_.N; a.f32 = env_.f32;
        a.epi = spec_.softcap > 0 ? lm::kEpiSoftcap : lm::kEpiNone;
        a.softcap = (float)spec_.softcap;
        return lm::linear(a, st);
    }
    ModelSpec spec_;
    Env env_;
    Work w_;
    std::vector<Layer> layers_;
    Mat embed_, head_;
    float *final_norm_ = nullptr, *x_ = nullptr;
};

int LayeredModel::load(DecodeContext& ctx, const std::string& dir) {
    if (!read_model_spec(dir, &spec_, &ctx.error)) return -3;
    bw_decode_config& c = ctx.cfg;
    c.layers = (int)spec_.layers.size();
    c.hidden = spec_.width;
    c.vocab = spec_.vocab;
    c.eps = (float)spec_.eps;
    env_.f32 = c.compute_f32;
    env_.slots = c.batch;
    env_.max_seq = c.max_seq;
    env_.width = spec_.width;
    env_.eps = (float)spec_.eps;
    env_.sms = sm_count(current_device());
    env_.max_rows = std::min(c.max_seq, c.max_portion > 0 ? c.max_portion : env_.f32 ? 512 : 4096);
    Loader l(ctx);
    if (!l.st.open(dir + "/model.safetensors", &ctx.error)) return -1;
    BW_TRY(l.matrix("embed", spec_.vocab, spec_.width, &embed_));
    BW_TRY(l.matrix("head", spec_.vocab, spec_.width, &head_));
    auto norm = [&](const std::string& name, float** dev) { return l.vec(name, {spec_.width}, dev, spec_.norm_offset); };
    BW_TRY(norm("final.norm", &final_norm_));
    layers_.resize(spec_.layers.size());
    for (size_t i = 0; i < layers_.size(); ++i) {
        const LayerSpec& s = spec_.layers[i];
        Layer& L = layers_[i];
        const std::string p = "l" + std::to_string(i) + ".";
        switch (s.mixer.kind) {
            case MixerSpec::kMamba2: L.mixer.reset(new Mamba2(s.mixer)); break;
            case MixerSpec::kRetention: L.mixer.reset(new Retention(s.mixer)); break;
            case MixerSpec::kLatentAttention:
                L.mixer.reset(new LatentAttention(
                    s.mixer, s.mixer.kv_from >= 0 ? static_cast<LatentAttention*>(layers_[s.mixer.kv_from].mixer.get()) : nullptr));
                break;
            case MixerSpec::kDelta: L.mixer.reset(new GatedDelta(s.mixer)); break;
            case MixerSpec::kDiffAttention:
                L.mixer.reset(new DiffAttention(
                    s.mixer, s.mixer.kv_from >= 0 ? static_cast<DiffAttention*>(layers_[s.mixer.kv_from].mixer.get()) : nullptr));
                break;
        }
        BW_TRY(L.mixer->load(l, p + "mix.", spec_.width));
        if (spec_.input_norms) BW_TRY(norm(p + "norm1", &L.in1));
        BW_TRY(norm(p + (spec_.input_norms ? "norm1b" : "norm1"), &L.out1));
        L.ff = s.ff;
        if (s.ff > 0) {
            if (spec_.input_norms) BW_TRY(norm(p + "norm2", &L.in2));
            BW_TRY(norm(p + (spec_.input_norms ? "norm2b" : "norm2"), &L.out2));
            std::vector<uint16_t> g, u;
            BW_TRY(l.tensor(p + "mlp.gate", {s.ff, spec_.width}, &g));
            BW_TRY(l.tensor(p + "mlp.up", {s.ff, spec_.width}, &u));
            Stack st(spec_.width);
            st.grow(2 * s.ff);
            for (int j = 0; j < s.ff; ++j) {   // interleaved: the product's epilogue sees gate j beside up j
                std::copy_n(&g[(size_t)j * spec_.width], spec_.width, st.row(2 * j));
                std::copy_n(&u[(size_t)j * spec_.width], spec_.width, st.row(2 * j + 1));
            }
            BW_TRY(l.upload(st, &L.gu));
            BW_TRY(l.matrix(p + "mlp.down", spec_.width, s.ff, &L.down));
        }
    }
    return 0;
}

int LayeredModel::alloc_state(DecodeContext& ctx) {
    // cos / sin of every rotation in use, computed in double precision
    std::map<Rotation, float2*> tables;
    for (Layer& L : layers_) {
        if (L.mixer->rotates()) {
            const Rotation& rot = L.mixer->spec().rot;
            const int half = rot.dims / 2;
            float2*& t = tables[rot];
            if (!t) {
                std::vector<float2> h((size_t)std::max(1, half) * env_.max_seq);
                const double gain = rot.gain();
                for (int i = 0; i < half; ++i) {
                    const double f = rot.frequency(i);
                    for (int p = 0; p < env_.max_seq; ++p)
                        h[(size_t)p * half + i] = make_float2((float)(cos(p * f) * gain), (float)(sin(p * f) * gain));
                }
                BW_TRY(ctx.upload(&t, h));
            }
            L.mixer->set_rotation(t);
        }
        BW_TRY(L.mixer->alloc(ctx, env_, &w_));
        w_.ff = std::max(w_.ff, (long)pad8(L.ff));
    }
    const size_t rows = std::max(env_.max_rows, env_.slots), el = env_.elem();
    w_.ldx = pad8(env_.width);
    auto act = [&](void** p, size_t elems) {
        char* c = nullptr;
        BW_TRY(ctx.alloc(&c, std::max<size_t>(elems, 8) * el));
        *p = c;
        return (int)cudaMemset(c, 0, std::max<size_t>(elems, 8) * el);
    };
    BW_TRY(act(&w_.xb, rows * w_.ldx));
    BW_TRY(act(&w_.proj_b, rows * w_.proj));
    BW_TRY(act(&w_.conv_b, rows * w_.conv));
    BW_TRY(act(&w_.mixed_b, rows * w_.mixed));
    BW_TRY(act(&w_.ff_b, rows * w_.ff));
    BW_TRY(act(&w_.fin_b, (size_t)std::max(kLogitRows, env_.slots) * w_.ldx));
    BW_TRY(act(&w_.kv_b, w_.kv));
    BW_TRY(ctx.alloc(&w_.proj32_b, rows * w_.proj32));
    BW_TRY(ctx.alloc(&w_.o32_b, rows * w_.o32));
    BW_TRY(ctx.alloc(&w_.log_decay, rows * w_.heads));
    BW_TRY(ctx.alloc(&w_.weight, rows * w_.heads));
    BW_TRY(ctx.alloc(&w_.sub, rows * env_.width));
    BW_TRY(ctx.alloc(&w_.part_b, w_.part));
    char* q = nullptr;
    BW_TRY(ctx.alloc(&q, w_.absorbed_bytes));
    w_.qabs_b = q;
    BW_TRY(ctx.alloc(&q, w_.chunk_bytes));
    w_.chunk_b = q;
    BW_TRY(ctx.alloc(&x_, rows * env_.width));
    ctx.x = x_;
    return ctx.alloc(&ctx.logits, (size_t)env_.slots * spec_.vocab);
}

int LayeredModel::enqueue_layers(DecodeContext& ctx, const lm::Rows& r, const int* tokens, cudaStream_t st) {
    const Env& e = env_;
    BW_TRY(lm::embed(x_, w_.xb, w_.ldx, embed_.p, embed_.ld, tokens, r.T, e.width, spec_.vocab, (float)spec_.embed_scale, layers_[0].in1,
                     e.eps, e.f32, st));
    for (size_t i = 0; i < layers_.size(); ++i) {
        Layer& L = layers_[i];
        const float* next = i + 1 < layers_.size() ? layers_[i + 1].in1 : nullptr;   // the next layer's input norm
        lm::LinearArgs a{};
        a.T = r.T; a.f32 = e.f32; a.y = w_.sub; a.ldy = e.width; a.y_f32 = 1; a.N = a.split = e.width;
        BW_TRY(L.mixer->run(e, w_, r, st));
        const Mat& o = L.mixer->out();
        a.x = w_.mixed_b; a.ldx = L.mixer->mixed_ld(); a.W = o.p; a.ldw = o.ld; a.K = o.K;
        BW_TRY(lm::linear(a, st));
        BW_TRY(lm::norm_add(x_, w_.xb, w_.ldx, w_.sub, L.out1, L.ff > 0 ? L.in2 : next, r.T, e.width, e.eps, e.f32, st));
        if (L.ff > 0) {
            lm::LinearArgs g{};
            g.x = w_.xb; g.ldx = w_.ldx; g.W = L.gu.p; g.ldw = L.gu.ld; g.T = r.T; g.N = g.split = L.gu.N; g.K = L.gu.K;
            g.y = w_.ff_b; g.ldy = pad8(L.ff); g.epi = lm::kEpiSwiglu; g.f32 = e.f32;
            BW_TRY(lm::linear(g, st));
            a.x = w_.ff_b; a.ldx = pad8(L.ff); a.W = L.down.p; a.ldw = L.down.ld; a.K = L.down.K;
            BW_TRY(lm::linear(a, st));
            BW_TRY(lm::norm_add(x_, w_.xb, w_.ldx, w_.sub, L.out2, next, r.T, e.width, e.eps, e.f32, st));
        }
        if (ctx.watch)
            BW_TRY(cudaMemcpyAsync(ctx.watch + ((size_t)i * ctx.watch_rows + ctx.watch_row0) * e.width, x_, (size_t)r.T * e.width * 4,
                                   cudaMemcpyDeviceToDevice, st));
    }
    return 0;
}

}  // namespace

std::unique_ptr<DecodeModel> make_layered_model() { return std::unique_ptr<DecodeModel>(new LayeredModel()); }

}  // namespace bw
