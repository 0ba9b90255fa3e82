// Batched decode driver: slots, positions, prompt tables, sampling, and the step as a CUDA graph, over a model family
// (decode_model.h).  The token loop is that of the INT4 servers (server/inference_server_int4_batched.cu:253-298) in the
// graph form of bench/decode_int4_cgraph_8b.cu:249-399 (stream capture, instantiate, launch per step): per-sequence
// positions and token bookkeeping live in device memory, and ONE CUDA graph per step is captured at creation and only
// replayed afterwards -- no allocation, no host-device synchronisation and no host decision inside a generation.
//
// Families that take portions (several consecutive tokens of one sequence at once) have their prompts filled in by
// bw_decode_begin that way, so that the graph's steps only generate; bw_decode_portion feeds tokens of one slot directly.
#include <cuda_runtime.h>
#include <stdint.h>
#include <stdio.h>
#include <string.h>

#include <algorithm>
#include <new>
#include <string>
#include <vector>

#include "decode_model.h"

struct bw_decode {
    bw::DecodeContext ctx;
    std::unique_ptr<bw::DecodeModel> model;
    int *sampled = nullptr, *prompt = nullptr, *prompt_len = nullptr, *gen = nullptr;
    int max_prompt = 0, max_new = 0;
    // portions: tokens, wanted rows, logits of a block of wanted rows, {slot, position} of a single token
    int *p_tokens = nullptr, *p_want = nullptr, *p_one = nullptr;
    float* p_logits = nullptr;
    std::vector<int> at;   // tokens every slot holds, as the host knows them
    cudaStream_t cap_stream = nullptr;
    cudaGraph_t graph = nullptr;
    cudaGraphExec_t exec = nullptr;
};

namespace {

constexpr int kWantRows = 64;   // logit rows copied to the host per block

int enqueue_step(bw_decode* d, cudaStream_t st) {
    bw::DecodeContext& c = d->ctx;
    const int M = c.cfg.batch;
    BW_TRY(bw_select_input_tokens(c.tokens_in, d->sampled, d->prompt, d->prompt_len, c.pos, M, d->max_prompt, st));
    BW_TRY(d->model->enqueue_tokens(c, M, c.slots, c.pos, c.tokens_in, c.logits, st));
    BW_TRY(bw_sample_argmax_batched(c.logits, c.cfg.vocab, c.cfg.vocab, M, d->sampled, c.pos, c.cfg.max_seq - 1, st));
    BW_TRY(bw_record_generated(d->gen, d->sampled, d->prompt_len, c.pos, M, d->max_new, st));
    return 0;
}

int alloc_driver(bw_decode* d) {
    bw::DecodeContext& c = d->ctx;
    const size_t M = c.cfg.batch;
    std::vector<int> ids(M);
    for (size_t m = 0; m < M; ++m) ids[m] = (int)m;
    d->max_prompt = c.cfg.max_prompt > 0 ? c.cfg.max_prompt : 1;
    d->max_new = c.cfg.max_new > 0 ? c.cfg.max_new : 1;
    BW_TRY(c.upload(&c.slots, ids));
    auto zeroed = [&](int** p, size_t n) {
        BW_TRY(c.alloc(p, n));
        return (int)cudaMemset(*p, 0, n * 4);
    };
    BW_TRY(zeroed(&c.tokens_in, M));
    BW_TRY(zeroed(&c.pos, M));
    BW_TRY(zeroed(&d->sampled, M));
    BW_TRY(zeroed(&d->prompt_len, M));
    BW_TRY(zeroed(&d->prompt, M * (size_t)d->max_prompt));
    BW_TRY(zeroed(&d->gen, M * (size_t)d->max_new));
    d->at.assign(M, 0);
    if (d->model->max_portion() > 0) {
        BW_TRY(zeroed(&d->p_tokens, d->model->max_portion()));
        BW_TRY(zeroed(&d->p_want, d->model->max_portion()));
        BW_TRY(zeroed(&d->p_one, 2));
        BW_TRY(c.alloc(&d->p_logits, (size_t)kWantRows * c.cfg.vocab));
    }
    return 0;
}

// Tokens of one slot, `tokens` in device memory: portions of at most max_portion.
int feed(bw_decode* d, int slot, const int* tokens, int n, cudaStream_t st) {
    for (int i = 0; i < n;) {
        const int len = std::min(n - i, d->model->max_portion());
        BW_TRY(d->model->enqueue_portion(d->ctx, slot, d->at[slot], len, tokens + i, 0, nullptr, nullptr, st));
        d->at[slot] += len;
        i += len;
    }
    return 0;
}

}  // namespace

extern "C" int bw_decode_create(const bw_decode_config* cfg, bw_decode** out) {
    if (!cfg || !out) return cudaErrorInvalidValue;
    *out = nullptr;
    if (cfg->batch < 1 || cfg->batch > 256 || cfg->max_seq < 1 || !cfg->weights_dir) return cudaErrorInvalidValue;
    bw_decode* d = new (std::nothrow) bw_decode();
    if (!d) return cudaErrorMemoryAllocation;
    const std::string dir = cfg->weights_dir;
    d->ctx.cfg = *cfg;
    d->ctx.cfg.weights_dir = nullptr;  // not kept beyond this call
    d->model = bw::make_decode_model(dir);
    if (!d->model) d->ctx.error = dir + ": not a model this program serves";
    int e = d->model ? d->model->load(d->ctx, dir) : (int)cudaErrorInvalidValue;
    if (e == 0) e = d->model->alloc_state(d->ctx);
    if (e == 0) e = alloc_driver(d);
    // One eager step sizes the library's scratch memory (the capture below must not allocate), then the step is
    // captured once; afterwards bw_decode_step only replays the graph.
    if (e == 0) e = (int)cudaStreamCreateWithFlags(&d->cap_stream, cudaStreamNonBlocking);
    if (e == 0) e = (int)cudaDeviceSynchronize();
    if (e == 0) e = enqueue_step(d, d->cap_stream);
    if (e == 0) e = (int)cudaStreamSynchronize(d->cap_stream);
    if (e == 0 && cfg->use_graph) {
        e = (int)cudaStreamBeginCapture(d->cap_stream, cudaStreamCaptureModeThreadLocal);
        if (e == 0) {
            const int se = enqueue_step(d, d->cap_stream);
            const int ee = (int)cudaStreamEndCapture(d->cap_stream, &d->graph);
            e = se ? se : ee;
        }
        if (e == 0) e = (int)cudaGraphInstantiate(&d->exec, d->graph, 0);
    }
    if (e == 0) e = (int)cudaMemset(d->ctx.pos, 0, (size_t)cfg->batch * 4);
    if (e == 0) e = (int)cudaDeviceSynchronize();
    if (e != 0) {
        if (!d->ctx.error.empty()) fprintf(stderr, "bw_decode_create: %s\n", d->ctx.error.c_str());
        bw_decode_destroy(d);
        return e;
    }
    *out = d;
    return 0;
}

extern "C" int bw_decode_get_config(const bw_decode* d, bw_decode_config* out) {
    if (!d || !out) return cudaErrorInvalidValue;
    *out = d->ctx.cfg;
    return 0;
}

extern "C" int bw_decode_begin(bw_decode* d, const int* prompt_ids, const int* prompt_len, int max_prompt, void* stream) {
    if (!d || !prompt_ids || !prompt_len || max_prompt < 1 || max_prompt > d->max_prompt) return cudaErrorInvalidValue;
    const int M = d->ctx.cfg.batch;
    const bool portions = d->model->max_portion() > 0;
    for (int m = 0; m < M; ++m)
        if (prompt_len[m] < 1 || prompt_len[m] > max_prompt || (portions && prompt_len[m] > d->ctx.cfg.max_seq)) return cudaErrorInvalidValue;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    // the device-side table has rows of d->max_prompt ids
    std::vector<int> table((size_t)M * d->max_prompt, 0);
    for (int m = 0; m < M; ++m) memcpy(&table[(size_t)m * d->max_prompt], prompt_ids + (size_t)m * max_prompt, (size_t)max_prompt * 4);
    BW_TRY(cudaMemcpyAsync(d->prompt, table.data(), table.size() * 4, cudaMemcpyHostToDevice, st));
    BW_TRY(cudaMemcpyAsync(d->prompt_len, prompt_len, (size_t)M * 4, cudaMemcpyHostToDevice, st));
    BW_TRY(cudaMemsetAsync(d->gen, 0xFF, (size_t)M * d->max_new * 4, st));  // -1 = not generated
    d->at.assign(M, 0);
    if (portions)   // everything but the last prompt token, which the first step takes
        for (int m = 0; m < M; ++m) BW_TRY(feed(d, m, d->prompt + (size_t)m * d->max_prompt, prompt_len[m] - 1, st));
    BW_TRY(cudaMemcpyAsync(d->ctx.pos, d->at.data(), (size_t)M * 4, cudaMemcpyHostToDevice, st));
    return (int)cudaStreamSynchronize(st);  // the pageable host buffers above must outlive the copies
}

extern "C" int bw_decode_steps(const bw_decode* d, int longest_prompt, int new_tokens) {
    if (!d || longest_prompt < 1 || new_tokens < 1) return 0;
    return d->model->max_portion() > 0 ? new_tokens : longest_prompt + new_tokens - 1;
}

extern "C" int bw_decode_step(bw_decode* d, void* stream) {
    if (!d) return cudaErrorInvalidValue;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    for (int& p : d->at) p = std::min(p + 1, std::max(p, d->ctx.cfg.max_seq - 1));
    if (d->exec) return (int)cudaGraphLaunch(d->exec, st);
    return enqueue_step(d, st);
}

extern "C" int bw_decode_portion(bw_decode* d, int slot, const int* tokens, int n, const int* want, int n_want, float* logits_out,
                                 void* stream) {
    if (!d || !tokens || n < 1 || n_want < 0 || (n_want > 0 && (!want || !logits_out))) return cudaErrorInvalidValue;
    const bw_decode_config& c = d->ctx.cfg;
    if (d->model->max_portion() < 1) return cudaErrorNotSupported;
    if (slot < 0 || slot >= c.batch || d->at[slot] + n > c.max_seq) return cudaErrorInvalidValue;
    for (int i = 0; i < n; ++i)
        if (tokens[i] < 0 || tokens[i] >= c.vocab) return cudaErrorInvalidValue;
    for (int i = 0; i < n_want; ++i)
        if (want[i] < 0 || want[i] >= n || (i > 0 && want[i] <= want[i - 1])) return cudaErrorInvalidValue;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    int w = 0;
    for (int i = 0; i < n;) {
        const int len = std::min(n - i, d->model->max_portion());
        std::vector<int> rows;
        while (w + (int)rows.size() < n_want && want[w + rows.size()] < i + len) rows.push_back(want[w + rows.size()] - i);
        d->ctx.watch_row0 = i;
        BW_TRY(cudaMemcpyAsync(d->p_tokens, tokens + i, (size_t)len * 4, cudaMemcpyHostToDevice, st));
        if (len == 1) {   // one token: the decode step's kernels
            const int one[2] = {slot, d->at[slot]};
            BW_TRY(cudaMemcpyAsync(d->p_one, one, 8, cudaMemcpyHostToDevice, st));
            BW_TRY(d->model->enqueue_tokens(d->ctx, 1, d->p_one, d->p_one + 1, d->p_tokens, d->p_logits, st));
            if (!rows.empty())
                BW_TRY(cudaMemcpyAsync(logits_out + (size_t)w * c.vocab, d->p_logits, (size_t)c.vocab * 4, cudaMemcpyDeviceToHost, st));
            BW_TRY(cudaStreamSynchronize(st));
        } else {
            BW_TRY(cudaMemcpyAsync(d->p_want, rows.data(), rows.size() * 4, cudaMemcpyHostToDevice, st));
            BW_TRY(d->model->enqueue_portion(d->ctx, slot, d->at[slot], len, d->p_tokens, 0, nullptr, nullptr, st));
            for (size_t b = 0; b < rows.size(); b += kWantRows) {
                const int nb = (int)std::min<size_t>(kWantRows, rows.size() - b);
                BW_TRY(d->model->enqueue_portion(d->ctx, slot, d->at[slot], 0, nullptr, nb, d->p_want + b, d->p_logits, st));
                BW_TRY(cudaMemcpyAsync(logits_out + (size_t)(w + b) * c.vocab, d->p_logits, (size_t)nb * c.vocab * 4, cudaMemcpyDeviceToHost, st));
            }
            BW_TRY(cudaStreamSynchronize(st));
        }
        d->at[slot] += len;
        w += (int)rows.size();
        i += len;
    }
    return cudaMemcpy(d->ctx.pos + slot, &d->at[slot], 4, cudaMemcpyHostToDevice);
}

extern "C" int bw_decode_release(bw_decode* d, int slot) {
    if (!d || slot < 0 || slot >= d->ctx.cfg.batch) return cudaErrorInvalidValue;
    d->at[slot] = 0;
    return cudaMemcpy(d->ctx.pos + slot, &d->at[slot], 4, cudaMemcpyHostToDevice);
}

extern "C" int bw_decode_held(const bw_decode* d, int slot) {
    return d && slot >= 0 && slot < d->ctx.cfg.batch ? d->at[slot] : -1;
}

extern "C" int bw_decode_watch_layers(bw_decode* d, float* buffer, long rows) {
    if (!d || (buffer && rows < 1)) return cudaErrorInvalidValue;
    d->ctx.watch = buffer;
    d->ctx.watch_rows = rows;
    d->ctx.watch_row0 = 0;
    return 0;
}

extern "C" int bw_decode_result(bw_decode* d, int* gen_out, void* stream) {
    if (!d || !gen_out) return cudaErrorInvalidValue;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    BW_TRY(cudaMemcpyAsync(gen_out, d->gen, (size_t)d->ctx.cfg.batch * d->max_new * 4, cudaMemcpyDeviceToHost, st));
    return (int)cudaStreamSynchronize(st);
}

extern "C" int bw_decode_buffers(bw_decode* d, float** logits, float** hidden, int** positions, int** sampled,
                                 uint16_t** k_cache, uint16_t** v_cache) {
    if (!d) return cudaErrorInvalidValue;
    uint16_t *k = nullptr, *v = nullptr;
    d->model->caches(&k, &v);
    if (logits) *logits = d->ctx.logits;
    if (hidden) *hidden = d->ctx.x;
    if (positions) *positions = d->ctx.pos;
    if (sampled) *sampled = d->sampled;
    if (k_cache) *k_cache = k;
    if (v_cache) *v_cache = v;
    return 0;
}

extern "C" int bw_decode_destroy(bw_decode* d) {
    if (!d) return cudaErrorInvalidValue;
    cudaDeviceSynchronize();
    if (d->exec) cudaGraphExecDestroy(d->exec);
    if (d->graph) cudaGraphDestroy(d->graph);
    if (d->cap_stream) cudaStreamDestroy(d->cap_stream);
    for (void* p : d->ctx.owned) cudaFree(p);
    delete d;
    return 0;
}
