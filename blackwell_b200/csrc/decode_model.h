// Interface between the decode driver (bw_decode_*: slots, positions, prompt tables, graph, sampling) and a model family.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#include <memory>
#include <string>
#include <vector>

#include "../../include/blackwell_b200.h"

namespace bw {

#define BW_TRY(expr)                       \
    do {                                   \
        const int e_ = (int)(expr);        \
        if (e_ != 0) return e_;            \
    } while (0)

// What the driver and its model share.
struct DecodeContext {
    bw_decode_config cfg;
    std::string error;            // why creation failed, printed by the driver
    std::vector<void*> owned;     // every device allocation, for teardown
    // token bookkeeping of the driver, one entry per sequence
    int *tokens_in = nullptr, *pos = nullptr, *slots = nullptr;   // slots: 0, 1, ... batch - 1
    float *x = nullptr, *logits = nullptr;                        // set by the model: hidden state, logits [batch][vocab]
    float* watch = nullptr;       // optional: residual stream after every layer of a portion, [layers][rows][hidden]
    long watch_rows = 0, watch_row0 = 0;

    template <typename T>
    int alloc(T** p, size_t count) {
        void* v = nullptr;
        cudaError_t e = cudaMalloc(&v, count * sizeof(T) ? count * sizeof(T) : 1);
        if (e != cudaSuccess) return (int)e;
        owned.push_back(v);
        *p = static_cast<T*>(v);
        return 0;
    }
    template <typename T>
    int upload(T** p, const std::vector<T>& h) {
        BW_TRY(alloc(p, h.size()));
        return (int)cudaMemcpy(*p, h.data(), h.size() * sizeof(T), cudaMemcpyHostToDevice);
    }
};

class DecodeModel {
public:
    virtual ~DecodeModel() {}
    // Checks (or fills in) the sizes in ctx.cfg, reads the weights, uploads them.
    virtual int load(DecodeContext& ctx, const std::string& dir) = 0;
    // Caches, states and work buffers; sets ctx.x and ctx.logits.
    virtual int alloc_state(DecodeContext& ctx) = 0;
    // One token per row: row m continues the sequence in slot slots[m] at position pos[m] with token tokens[m] (device
    // arrays); logits [rows][vocab].
    virtual int enqueue_tokens(DecodeContext& ctx, int rows, const int* slots, const int* pos, const int* tokens, float* logits,
                               cudaStream_t st) = 0;
    // Most consecutive tokens of one sequence per call of enqueue_portion; 0: the family takes tokens one by one only.
    virtual int max_portion() const { return 0; }
    // tokens [n] of the sequence in `slot` at pos0, pos0 + 1, ...; logits [n_want][vocab] of the rows want [n_want] (device).
    virtual int enqueue_portion(DecodeContext&, int, int, int, const int*, int, const int*, float*, cudaStream_t) {
        return cudaErrorNotSupported;
    }
    virtual void caches(uint16_t** k, uint16_t** v) { *k = *v = nullptr; }
};

std::unique_ptr<DecodeModel> make_layered_model();   // directories with a config.json
std::unique_ptr<DecodeModel> make_int4_model();      // the INT4 container format (sizes given by the caller)

// The family of a weight directory.
std::unique_ptr<DecodeModel> make_decode_model(const std::string& dir);

}  // namespace bw
