// Operations of the config.json models (bfloat16 weights): launch interfaces shared by the layered model and the C
// entry points.  Activations are bfloat16 (serving) or fp32 (32-bit mode); the residual stream, norms, attention
// scores, decays and recurrent states are fp32 in both.  Row strides are in elements.  Per-head blocks are padded to
// multiples of eight columns (pad8), so that every row of every operand starts on a 16-byte boundary.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace bw {
namespace lm {

typedef __nv_bfloat16 bf16;

inline __host__ __device__ int pad8(int n) { return (n + 7) & ~7; }
inline __host__ __device__ int pad16(int n) { return (n + 15) & ~15; }

// ---------------------------------------------------------------- linear: y[t][n] = sum_k x[t][k] W[n][k]
enum : int { kEpiNone = 0, kEpiSwiglu = 1, kEpiSoftcap = 2 };
struct LinearArgs {
    const void* x;        // [T][ldx] bf16, or fp32 when f32 != 0
    long ldx;
    const bf16* W;        // [N][ldw], ldw a multiple of 8, zero beyond K
    long ldw;
    int T, N, K;
    void* y;              // columns below `split`: bf16 (fp32 when f32), stride ldy; swiglu: N/2 columns
    long ldy;
    int y_f32;            // y is fp32 in either mode
    float* y32;           // columns from `split` on, fp32, stride ldy32 (split == N: none)
    long ldy32;
    int split;
    int epi;              // kEpiSwiglu: rows 2j / 2j+1 of W are gate j / up j, y[j] = silu(gate) * up
    float softcap;        // kEpiSoftcap: y = softcap * tanh(y / softcap)
    int f32;
};
cudaError_t linear(const LinearArgs& a, cudaStream_t st);

// ---------------------------------------------------------------- rows of a step
// One token of each of M sequences (slot / pos in device memory), or T consecutive tokens of one sequence.
struct Rows {
    int T;                 // rows
    const int* row_slot;   // device, per row (token step); NULL: all rows belong to `slot`, at pos0, pos0 + 1, ...
    const int* row_pos;
    int slot, pos0;
    __device__ __forceinline__ int slot_of(int r) const { return row_slot ? row_slot[r] : slot; }
    __device__ __forceinline__ int pos_of(int r) const { return row_pos ? row_pos[r] : pos0 + r; }
};

// ---------------------------------------------------------------- embedding, norms
// xb = norm(x) * next in the activation type, or x itself where next is NULL: the next sublayer's input.
// x <- table[token] * scale
cudaError_t embed(float* x, void* xb, long ldxb, const bf16* table, long ldt, const int* tokens, int T, int width, int vocab,
                  float scale, const float* next, float eps, int f32, cudaStream_t st);
// x <- x + y / sqrt(mean y^2 + eps) * w
cudaError_t norm_add(float* x, void* xb, long ldxb, const float* y, const float* w, const float* next, int T, int width, float eps,
                     int f32, cudaStream_t st);
// xb = x / sqrt(mean x^2 + eps) * w for the rows listed in `rows` (NULL: all)
cudaError_t norm_rows(void* xb, long ldxb, const float* x, const float* w, const int* rows, int T, int width, float eps, int f32,
                      cudaStream_t st);
// Gated norm over `groups` equal parts of the heads * V channels (head h's channels start at column h * pad8(V)):
//   gate_first: u = o * silu(g), out = u / rms(u) * w;   otherwise: out = o / rms(o) * w * silu(g).   w may be NULL (= 1).
cudaError_t gated_norm(void* out, long ldout, const float* o, long ldo, const void* gate, long ldg, const float* w, int T,
                       int heads, int V, int groups, int gate_first, float eps, int f32, cudaStream_t st);

// ---------------------------------------------------------------- short causal convolution + silu, step sizes
struct ConvArgs {
    const void* u;          // projection rows: channel c (conv order) at column off_x + padded position
    long ldu;
    const float* w;         // [channels][taps]
    const float* bias;      // [channels] or NULL
    float* ring;            // [slot][taps][channels] last inputs, entry = position % taps
    int taps, heads, V, N, groups;   // channels: heads * V, then groups * N (k), then groups * N (q)
    int off;                // first padded column of the convolved part in u
    void* out;              // [T][ldo] same padded layout, columns from 0
    long ldo;
    const float* dt_raw;    // [T][ld_dt]
    long ld_dt;
    const float *dt_bias, *A_log;    // [heads]
    const float* beta_raw;           // [T][ld_dt] or NULL: the weight is sigmoid(beta_raw) instead of the step size
    float *log_decay, *weight;       // [T][heads]
};
cudaError_t conv_silu(const ConvArgs& c, const Rows& r, int f32, cudaStream_t st);     // several rows of one sequence
cudaError_t conv_ring_store(const ConvArgs& c, const Rows& r, int f32, cudaStream_t st);  // after conv_silu

// ---------------------------------------------------------------- gated linear recurrence
//   S_t = exp(log_decay_t) S_(t-1) + weight_t k_t v_t^T,   o_t = S_t^T q_t + D v_t        (per head; S is N x V, fp32)
// Delta rule (`delta`): k and q enter as unit vectors, x / sqrt(sum x^2 + unit_eps), q times q_scale, and what is written is the
// part of v_t that the decayed state does not hold yet:
//   S_t = S' + k_t u_t^T  with  S' = exp(log_decay_t) S_(t-1),  u_t = weight_t (v_t - S'^T k_t),   o_t = S_t^T q_t
struct RecurrenceArgs {
    const void *q, *k, *v;           // q/k of head h at column (h / (heads / groups)) * pad8(N), v at h * pad8(V)
    long ldq, ldk, ldv;
    int heads, N, V, groups;
    const float *log_decay, *weight;  // [T][heads] or NULL
    const float* head_log_decay;      // [heads], used when log_decay is NULL (weight_t = const_weight then)
    float const_weight;
    const float* D;                   // [heads] or NULL
    float* S;                         // [slot][heads][N][pad8(V)]
    float* o;                         // [T][ldo], head h at column h * pad8(V)
    long ldo;
    int delta;                        // log_decay and weight are given, D is not
    float unit_eps, q_scale;
    void* chunk_scratch;              // delta_chunk_bytes, delta chunks only
};
// `conv` != NULL (one row per sequence): q, k, v and the decays come from the projection through the convolution.
cudaError_t recurrence_step(const RecurrenceArgs& a, const ConvArgs* conv, const Rows& r, int f32, cudaStream_t st);
bool recurrence_chunk_supported(const RecurrenceArgs& a);
cudaError_t recurrence_chunk(const RecurrenceArgs& a, const Rows& r, cudaStream_t st);   // bf16, rows of one sequence
size_t delta_chunk_bytes(int rows, int heads);
bool delta_chunk_supported(const RecurrenceArgs& a);
cudaError_t delta_chunk(const RecurrenceArgs& a, const Rows& r, cudaStream_t st);        // bf16, rows of one sequence

// ---------------------------------------------------------------- latent attention
constexpr int kPartStats = 4;   // floats after a split's outputs: running maximum, sum, padding
struct LatentArgs {
    int heads, dim, rot, V, R;        // per head: unrotated / rotated query size, value size; latent size
    int rot_dims;                     // rotated part of the `rot` dimensions
    float scale, eps;
    const float2* cs;                 // cos / sin [max_seq][rot_dims / 2]
    int max_seq;
    void* cache;                      // [slot][max_seq][ldc]: latent at 0, rotated key part at pad8(R)
    long ldc;
    void* q;                          // [T][ldq], head h at h * (pad8(dim) + pad8(rot)), rotated part at + pad8(dim)
    long ldq;
    const float* dkv;                 // [T][ld32] fp32 latent + key part (NULL: another layer's cache is read)
    const float* gate;                // [T][ld32] fp32 gate logits, one per head
    long ld32;
    const float* dkv_norm;            // [R]
    const bf16* Wkv;                  // rows: uk (head h at h * pad8(dim)), then uv (head h at heads * pad8(dim) + h * pad8(V))
    long ldw;                         // pad8(R)
    const float* sink;                // [heads]
    void* out;                        // [T][ldout], head h at h * pad8(V)
    long ldout;
    // scratch
    void* qabs;                       // [T][heads][2][Dp] bf16 (high, remainder) or [T][heads][Dp] fp32
    float* part;                      // [T][heads][splits][pad8(R) + kPartStats]
    int splits;
    void* kv;                         // expanded keys and values [max_seq][heads * (pad8(dim) + pad8(V))]
};
inline __host__ __device__ int latent_row(int R, int rot) { return pad8(R) + pad8(rot); }
inline __host__ __device__ int latent_dp(int R, int rot) { return pad16(pad8(R) + pad8(rot)); }
bool latent_absorbed_supported(const LatentArgs& a);
bool latent_expanded_supported(const LatentArgs& a);
// Absorbed form, any rows: queries go into the latent space, keys are the cache rows themselves.
cudaError_t latent_absorbed(const LatentArgs& a, const Rows& r, int f32, cudaStream_t st);
// Expanded form, rows of one sequence, bf16: keys and values of the whole context through Wkv, then flash attention.
cudaError_t latent_expanded(const LatentArgs& a, const Rows& r, cudaStream_t st);

// ---------------------------------------------------------------- differential attention
// Two softmax maps per query head over the same values, causal, over the last `window` positions:
//   o = a1 - lambda a2,   out = o / sqrt(mean o^2 + eps) * out_scale        (per head, a_i = softmax(scale q_i k_i^T) v)
// Query head h reads key / value head h / (heads / kv_heads).  Rotated pairs are (i, i + rot_dims / 2).
struct DiffAttnArgs {
    int heads, kv_heads, dim, V;
    int window;                       // 0: all earlier positions
    int rot_dims;
    const float2* cs;                 // cos / sin [max_seq][rot_dims / 2]
    int max_seq;
    float scale, lambda, out_scale, eps;
    void* cache;                      // [slot][cap] rows of kv_heads * diff_row: position p at row p % cap
    int cap, slots;                   // cap: max_seq, or a multiple of 16 of at least window - 1 + the rows of a call
    void* q;                          // [T][ld], head h's map i at (2 h + i) * pad8(dim), not rotated yet; portions rotate in place
    const void *k, *v;                // [T][ld], laid out the same way / head g at g * pad8(V); NULL: already in the cache
    long ld;
    void* out;                        // [T][ldout], head h at h * pad8(V)
    long ldout;
    int splits;                       // context splits of a token step (a cluster of 1, 2, 4 or 8 blocks)
};
inline __host__ __device__ int diff_row(int dim, int V) { return 2 * pad8(dim) + pad8(V); }   // map 1 key, map 2 key, value
bool diff_attention_supported(const DiffAttnArgs& a);
int diff_attention_splits(const DiffAttnArgs& a, int rows, int f32);
cudaError_t diff_attention(const DiffAttnArgs& a, const Rows& r, int f32, cudaStream_t st);

}  // namespace lm
}  // namespace bw
