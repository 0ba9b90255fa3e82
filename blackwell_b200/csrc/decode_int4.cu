// The INT4 container family of the decode driver (Qwen3-shaped trees).
//
// It mirrors the reference's per-layer sequence (server/inference_server_int4_batched.cu:253-298: rmsnorm ->
// quantize -> q/k/v GEMV -> head norm, RoPE -> KV update -> attention -> quantize -> o GEMV -> residual -> rmsnorm ->
// quantize -> gate/up GEMV -> SwiGLU -> quantize -> down GEMV -> residual; then final norm, LM head, sampling) with the
// fusions of this library: 6 or 7 launches per layer for the whole batch.
//
// Weights: a directory in the reference's container format (<l>_self_attn.q_proj.int4_t / .scale_t ..., see
// weight_files.cu) -- q, k, v are concatenated by rows into one matrix, gate and up likewise; the INT4 embedding is
// dequantized to fp32 once, as the reference does (:196-217).  Activation format: 8 = int8 activations with binary16
// weight scales (the fast path), 4 = the reference's own arithmetic (INT4 activations by the quantize_int4 rule, fp32
// weight scales).  The KV cache is binary16.
#include <cuda_fp16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <string.h>

#include <string>
#include <vector>

#include "decode_model.h"

namespace bw {
namespace {

struct Mat {          // one (possibly concatenated) projection on the device
    int K = 0, N = 0;
    uint8_t* packed = nullptr;
    float* sc32 = nullptr;
    uint16_t* sc16 = nullptr;
};

struct Layer {
    Mat qkv, o, gu, down;
    float *rn_in = nullptr, *rn_post = nullptr, *qn = nullptr, *kn = nullptr;
};

class Int4Model : public DecodeModel {
public:
    int load(DecodeContext& ctx, const std::string& dir) override {
        const bw_decode_config& c = ctx.cfg;
        if (c.layers < 1 || c.hidden < 32 || c.hidden % 32 != 0 || c.inter < 32 || c.inter % 32 != 0 || c.n_q_heads < 1 ||
            c.n_kv_heads < 1 || c.n_q_heads % c.n_kv_heads != 0 || c.head_dim != 128 || c.vocab < 1 ||
            (c.act_bits != 4 && c.act_bits != 8) || c.compute_f32)
            return cudaErrorInvalidValue;
        return load_model(&ctx, dir);
    }
    int alloc_state(DecodeContext& ctx) override { return alloc_buffers(&ctx); }
    int enqueue_tokens(DecodeContext& ctx, int rows, const int*, const int* pos, const int* tokens, float* logits,
                       cudaStream_t st) override {
        if (rows != ctx.cfg.batch) return cudaErrorNotSupported;   // row m is slot m
        return enqueue_step(&ctx, pos, tokens, logits, st);
    }
    void caches(uint16_t** k, uint16_t** v) override { *k = kc; *v = vc; }

private:
    std::vector<Layer> layers;
    Mat lm;
    float* rn_final = nullptr;
    float* embed = nullptr;  // fp32 [vocab][H]
    uint16_t *kc = nullptr, *vc = nullptr;
    float *qkv = nullptr, *q = nullptr, *attn = nullptr, *gu = nullptr;
    int8_t* attn_q = nullptr;   // attention result block-16 quantized by the attention kernel (int8 mode, fused form)
    float* attn_qs = nullptr;
    // norm-pending hand-over (one sequence, int8 mode): the hidden state after O (a) and after down (b), quantized
    int8_t *pa_q = nullptr, *pb_q = nullptr;
    float *pa_s = nullptr, *pa_ss = nullptr, *pb_s = nullptr, *pb_ss = nullptr;
    size_t kv_layer = 0, kv_batch = 0;

    int load_model(DecodeContext* d, const std::string& dir);
    int gemv(const DecodeContext* d, const Mat& W, float* y, const float* residual, const float* x, const float* up, long x_stride,
             const float* norm_w, int N_rows, cudaStream_t st);
    int enqueue_step(DecodeContext* d, const int* pos, const int* tokens, float* logits, cudaStream_t st);
    int alloc_buffers(DecodeContext* d);
};

uint16_t f32_to_f16_bits(float f) {
    const __half h = __float2half_rn(f);
    uint16_t b;
    memcpy(&b, &h, 2);
    return b;
}

// Reads the listed projections of one layer and uploads them stacked by rows.
int load_stacked(DecodeContext* d, const std::string& dir, const std::vector<std::string>& names, int K_expect, Mat* out) {
    std::vector<uint8_t> packed;
    std::vector<float> scales;
    int N = 0;
    for (const std::string& nm : names) {
        const std::string prefix = dir + "/" + nm;
        int k = 0, n = 0;
        int e = bw_w4_file_dims(prefix.c_str(), &k, &n);
        if (e != 0) { d->error = "cannot read " + prefix + ".int4_t/.scale_t"; return e; }
        if (k != K_expect) { d->error = prefix + ": K does not match the model shape"; return -3; }
        const size_t pb = packed.size(), sb = scales.size();
        packed.resize(pb + (size_t)n * k / 2);
        scales.resize(sb + (size_t)n * (k / 16));
        e = bw_w4_file_read(prefix.c_str(), packed.data() + pb, scales.data() + sb, k, n);
        if (e != 0) { d->error = "cannot read " + prefix; return e; }
        N += n;
    }
    out->K = K_expect;
    out->N = N;
    BW_TRY(d->upload(&out->packed, packed));
    if (d->cfg.act_bits == 4) {
        BW_TRY(d->upload(&out->sc32, scales));
    } else {
        std::vector<uint16_t> h16(scales.size());
        for (size_t i = 0; i < scales.size(); ++i) h16[i] = f32_to_f16_bits(scales[i]);
        BW_TRY(d->upload(&out->sc16, h16));
    }
    return 0;
}

int load_f32(DecodeContext* d, const std::string& path, size_t n, size_t offset, size_t total, float** out) {
    std::vector<float> h(total);
    const int e = bw_f32_file_read(path.c_str(), h.data(), total);
    if (e != 0) { d->error = "cannot read " + path; return e; }
    std::vector<float> part(h.begin() + offset, h.begin() + offset + n);
    return d->upload(out, part);
}

int Int4Model::load_model(DecodeContext* d, const std::string& dir) {
    const bw_decode_config& c = d->cfg;
    const int H = c.hidden, Q = c.n_q_heads * 128, KV = c.n_kv_heads * 128, I = c.inter;
    layers.resize(c.layers);
    for (int l = 0; l < c.layers; ++l) {
        const std::string p = std::to_string(l) + "_";
        Layer& L = layers[l];
        BW_TRY(load_stacked(d, dir, {p + "self_attn.q_proj", p + "self_attn.k_proj", p + "self_attn.v_proj"}, H, &L.qkv));
        BW_TRY(load_stacked(d, dir, {p + "self_attn.o_proj"}, Q, &L.o));
        BW_TRY(load_stacked(d, dir, {p + "mlp.gate_proj", p + "mlp.up_proj"}, H, &L.gu));
        BW_TRY(load_stacked(d, dir, {p + "mlp.down_proj"}, I, &L.down));
        if (L.qkv.N != Q + 2 * KV || L.o.N != H || L.gu.N != 2 * I || L.down.N != H) {
            d->error = "layer " + std::to_string(l) + ": projection sizes do not match the model shape";
            return -3;
        }
        BW_TRY(load_f32(d, dir + "/" + p + "input_layernorm.f32", H, 0, H, &L.rn_in));
        BW_TRY(load_f32(d, dir + "/" + p + "post_attention_layernorm.f32", H, 0, H, &L.rn_post));
        // qk_norms.f32 holds, per layer, the q-head norm then the k-head norm (128 floats each)
        BW_TRY(load_f32(d, dir + "/qk_norms.f32", 128, (size_t)l * 256, (size_t)c.layers * 256, &L.qn));
        BW_TRY(load_f32(d, dir + "/qk_norms.f32", 128, (size_t)l * 256 + 128, (size_t)c.layers * 256, &L.kn));
    }
    BW_TRY(load_f32(d, dir + "/final_norm.f32", H, 0, H, &rn_final));
    BW_TRY(load_stacked(d, dir, {"lm_head"}, H, &lm));
    if (lm.N < c.vocab) { d->error = "lm_head has fewer rows than the vocabulary"; return -3; }
    // embedding: INT4 -> fp32 once, (nibble - 8) * scale
    {
        const std::string prefix = dir + "/embed_tokens";
        int k = 0, n = 0;
        int e = bw_w4_file_dims(prefix.c_str(), &k, &n);
        if (e != 0 || k != H || n < c.vocab) { d->error = "cannot use " + prefix; return e ? e : -3; }
        std::vector<uint8_t> packed((size_t)n * k / 2);
        std::vector<float> sc((size_t)n * (k / 16));
        e = bw_w4_file_read(prefix.c_str(), packed.data(), sc.data(), k, n);
        if (e != 0) { d->error = "cannot read " + prefix; return e; }
        std::vector<float> table((size_t)c.vocab * H);
        for (int r = 0; r < c.vocab; ++r)
            for (int kb = 0; kb < H / 16; ++kb) {
                const float s = sc[(size_t)r * (H / 16) + kb];
                for (int i = 0; i < 16; ++i) {
                    const uint8_t byte = packed[(size_t)r * H / 2 + (size_t)kb * 8 + i / 2];
                    const int nib = (i & 1) ? (byte >> 4) : (byte & 0x0F);
                    table[(size_t)r * H + kb * 16 + i] = (float)(nib - 8) * s;
                }
            }
        BW_TRY(d->upload(&embed, table));
    }
    return 0;
}

// y = W . quantize(prologue(x)) (+ residual) in the engine's activation format.
int Int4Model::gemv(const DecodeContext* d, const Mat& W, float* y, const float* residual, const float* x, const float* up, long x_stride,
         const float* norm_w, int N_rows, cudaStream_t st) {
    const bw_decode_config& c = d->cfg;
    if (c.act_bits == 4)
        return bw_gemv_int4_decode(y, 0, residual, x, up, x_stride, norm_w, c.eps, W.packed, W.sc32, W.K, N_rows, c.batch, st);
    return bw_gemv_w4a8_decode(y, 0, residual, x, up, x_stride, norm_w, c.eps, W.packed, W.sc16, W.K, N_rows, c.batch, st);
}

int Int4Model::enqueue_step(DecodeContext* d, const int* pos, const int* tokens, float* logits, cudaStream_t st) {
    const bw_decode_config& c = d->cfg;
    const int M = c.batch, H = c.hidden, nq = c.n_q_heads, nkv = c.n_kv_heads, I = c.inter;
    BW_TRY(bw_embed_gather_f32(d->x, embed, tokens, H, c.vocab, M, st));
    // One sequence in int8 mode (at 5..16 the same hand-over measured no faster than the prep launches): the O and down projections hand their result to the next GEMV already quantized, so
    // that no CTA of the QKV / gate+up / LM-head GEMVs has to quantize the hidden state (bw_gemv_w4a8_pending).
    const bool pending = M == 1 && c.act_bits == 8 && (nq / nkv == 4 || nq / nkv == 8) && H % 16 == 0;
    auto pend = [&](float* y, const float* res, const Mat& W, int N, const int8_t* xq, const float* xs, const float* xss,
                    const float* gate, const float* up, const float* next_w, int8_t* nq_, float* ns, float* nss) {
        bw_gemv_pending_args g{};
        g.y = y; g.residual = res; g.x_q = xq; g.x_scale = xs; g.x_block_sumsq = xss; g.eps = c.eps;
        g.gate = gate; g.up = up; g.W_packed = W.packed; g.W_scale_f16 = W.sc16; g.K = W.K; g.N = N;
        g.next_norm_w = next_w; g.next_q = nq_; g.next_scale = ns; g.next_block_sumsq = nss;
        g.M = M; g.x_stride = gate ? 2 * (long)I : 0;
        return bw_gemv_w4a8_pending(&g, st);
    };
    for (int l = 0; l < c.layers; ++l) {
        const Layer& L = layers[l];
        const size_t off = (size_t)l * kv_layer;
        if (pending && l > 0)
            BW_TRY(pend(qkv, nullptr, L.qkv, L.qkv.N, pb_q, pb_s, pb_ss, nullptr, nullptr, nullptr, nullptr, nullptr, nullptr));
        else
            BW_TRY(gemv(d, L.qkv, qkv, nullptr, d->x, nullptr, 0, L.rn_in, L.qkv.N, st));
        const bool fused = nq / nkv == 4 || nq / nkv == 8;
        const bool q8 = fused && c.act_bits == 8;   // the attention kernel quantizes its result for the O projection
        if (q8) {
            BW_TRY(bw_attention_decode_f16kv_fused_q8(nullptr, attn_q, attn_qs, qkv, L.qn, L.kn, kc, vc,
                                                      pos, c.max_seq, nq, nkv, 128, c.max_seq, M, kv_batch, off,
                                                      c.eps, c.rope_base, st));
        } else if (fused) {  // head norm + RoPE + KV write inside the tensor-core attention kernel
            BW_TRY(bw_attention_decode_f16kv_fused(attn, qkv, L.qn, L.kn, kc, vc, pos, c.max_seq, nq, nkv, 128,
                                                   c.max_seq, M, kv_batch, off, c.eps, c.rope_base, st));
        } else {
            BW_TRY(bw_qk_norm_rope_kv_f16(q, kc, vc, qkv, L.qn, L.kn, pos, nq, nkv, 128, c.max_seq, M,
                                          kv_batch, off, c.eps, c.rope_base, st));
            BW_TRY(bw_attention_decode_f16kv(attn, q, kc, vc, pos, c.max_seq, nq, nkv, 128, c.max_seq, M,
                                             kv_batch, off, st));
        }
        if (pending) {
            const float* next_w = l + 1 < c.layers ? layers[l + 1].rn_in : rn_final;
            BW_TRY(pend(d->x, d->x, L.o, H, attn_q, attn_qs, nullptr, nullptr, nullptr, L.rn_post, pa_q, pa_s, pa_ss));
            BW_TRY(pend(gu, nullptr, L.gu, 2 * I, pa_q, pa_s, pa_ss, nullptr, nullptr, nullptr, nullptr, nullptr, nullptr));
            BW_TRY(pend(d->x, d->x, L.down, H, nullptr, nullptr, nullptr, gu, gu + I, next_w, pb_q, pb_s, pb_ss));
            continue;
        }
        if (q8)
            BW_TRY(bw_gemv_w4a8_q8_decode(d->x, 0, d->x, attn_q, attn_qs, L.o.packed, L.o.sc16, L.o.K, H, M, st));
        else
            BW_TRY(gemv(d, L.o, d->x, d->x, attn, nullptr, 0, nullptr, H, st));
        BW_TRY(gemv(d, L.gu, gu, nullptr, d->x, nullptr, 0, L.rn_post, 2 * I, st));
        BW_TRY(gemv(d, L.down, d->x, d->x, gu, gu + I, 2 * (long)I, nullptr, H, st));
    }
    if (pending)
        BW_TRY(pend(logits, nullptr, lm, c.vocab, pb_q, pb_s, pb_ss, nullptr, nullptr, nullptr, nullptr, nullptr, nullptr));
    else
        BW_TRY(gemv(d, lm, logits, nullptr, d->x, nullptr, 0, rn_final, c.vocab, st));
    return 0;
}

int Int4Model::alloc_buffers(DecodeContext* d) {
    const bw_decode_config& c = d->cfg;
    const size_t M = c.batch, H = c.hidden;
    kv_layer = (size_t)c.n_kv_heads * c.max_seq * 128;
    kv_batch = (size_t)c.layers * kv_layer;
    BW_TRY(d->alloc(&kc, M * kv_batch));
    BW_TRY(d->alloc(&vc, M * kv_batch));
    BW_TRY(d->alloc(&d->x, M * H));
    BW_TRY(d->alloc(&qkv, M * (size_t)(c.n_q_heads + 2 * c.n_kv_heads) * 128));
    BW_TRY(d->alloc(&q, M * (size_t)c.n_q_heads * 128));
    BW_TRY(d->alloc(&attn, M * (size_t)c.n_q_heads * 128));
    BW_TRY(d->alloc(&attn_q, M * (size_t)c.n_q_heads * 128));
    BW_TRY(d->alloc(&attn_qs, M * (size_t)c.n_q_heads * 8));
    BW_TRY(d->alloc(&pa_q, M * H));  BW_TRY(d->alloc(&pb_q, M * H));
    BW_TRY(d->alloc(&pa_s, M * (H / 16 + 1)));  BW_TRY(d->alloc(&pa_ss, M * (H / 16 + 1)));
    BW_TRY(d->alloc(&pb_s, M * (H / 16 + 1)));  BW_TRY(d->alloc(&pb_ss, M * (H / 16 + 1)));
    BW_TRY(d->alloc(&gu, M * 2 * (size_t)c.inter));
    BW_TRY(d->alloc(&d->logits, M * (size_t)c.vocab));
    BW_TRY(cudaMemset(kc, 0, M * kv_batch * 2));
    BW_TRY(cudaMemset(vc, 0, M * kv_batch * 2));
    return 0;
}

}  // namespace

std::unique_ptr<DecodeModel> make_int4_model() { return std::unique_ptr<DecodeModel>(new Int4Model()); }

}  // namespace bw
