// Element-wise and per-row kernels of the config.json models: embedding lookup, norms on the sublayer output with the
// residual sum, gated group norm, short causal convolution with its step sizes.  fp32 arithmetic throughout; activations
// are read and written as bf16 (serving) or fp32 (32-bit mode).
#include <cuda_runtime.h>

#include <algorithm>

#include "host_util.h"
#include "lm_device.cuh"
#include "lm_ops.h"

namespace bw {
namespace lm {
namespace {

// Row kernels: a block per row, VEC neighbouring columns per access (4, or 1 for widths that are not a multiple of 4), the
// first KEEP vectors of a thread in registers.  Weights are fetched before the kernel waits for its predecessor.
template <int VEC, int KEEP>
struct RowVecs {
    static constexpr int kKeep = KEEP;
    float v[kKeep][VEC];
    static __device__ __forceinline__ int col(int j) { return (j * blockDim.x + threadIdx.x) * VEC; }
    static __device__ __forceinline__ void get(const float* p, float (&x)[VEC]) {
        if constexpr (VEC == 4) *reinterpret_cast<float4*>(x) = *reinterpret_cast<const float4*>(p);
        else x[0] = p[0];
    }
    static __device__ __forceinline__ void put(float* p, const float (&x)[VEC]) {
        if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = *reinterpret_cast<const float4*>(x);
        else p[0] = x[0];
    }
    static __device__ __forceinline__ void put(bf16* p, const float (&x)[VEC]) {
        if constexpr (VEC == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(x[0], x[1]), pack_bf16(x[2], x[3]));
        else p[0] = __float2bfloat16_rn(x[0]);
    }
    // p NULL, or beyond the row: `other`
    __device__ __forceinline__ void load(const float* p, int width, float other) {
#pragma unroll
        for (int j = 0; j < kKeep; ++j) {
#pragma unroll
            for (int e = 0; e < VEC; ++e) v[j][e] = other;
            if (p && col(j) < width) get(p + col(j), v[j]);
        }
    }
    __device__ __forceinline__ float squares() const {
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < kKeep; ++j)
#pragma unroll
            for (int e = 0; e < VEC; ++e) s = fmaf(v[j][e], v[j][e], s);
        return s;
    }
    // f(column) for the columns that are not kept
    template <typename F>
    static __device__ __forceinline__ void beyond(int width, F f) {
        for (int i = kKeep * blockDim.x * VEC + threadIdx.x; i < width; i += blockDim.x) f(i);
    }
};

// xb = x / rms(x) * next (next NULL: x) for the block's row x, of which `keep` holds the first values, `gain` those of next.
template <typename A, int VEC, int KEEP>
__device__ __forceinline__ void next_input(A* xb, const float* x, const float* next, const RowVecs<VEC, KEEP>& keep,
                                           const RowVecs<VEC, KEEP>& gain, int width, float eps, float* buf) {
    typedef RowVecs<VEC, KEEP> R;
    float f = 1.f;
    if (next) {
        float ss = keep.squares();
        R::beyond(width, [&](int i) { ss = fmaf(x[i], x[i], ss); });
        f = 1.0f / sqrtf(block_sum(ss, buf) / (float)width + eps);
    }
#pragma unroll
    for (int j = 0; j < R::kKeep; ++j)
        if (R::col(j) < width) {
            float v[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) v[e] = keep.v[j][e] * f * gain.v[j][e];
            R::put(xb + R::col(j), v);
        }
    R::beyond(width, [&](int i) { xb[i] = from_f<A>(x[i] * f * (next ? next[i] : 1.f)); });
}

template <typename A, int VEC, int KEEP>
__global__ void __launch_bounds__(512) embed_kernel(float* x, A* xb, long ldxb, const bf16* table, long ldt, const int* tokens,
                                                    int width, int vocab, float scale, const float* next, float eps) {
    __shared__ float buf[32];
    typedef RowVecs<VEC, KEEP> R;
    R gain, keep;
    gain.load(next, width, 1.f);
    pdl_trigger();
    pdl_wait();
    const long r = blockIdx.x;
    int tok = tokens[r];
    tok = tok < 0 ? 0 : tok >= vocab ? vocab - 1 : tok;
    const bf16* row = table + (long)tok * ldt;
    float* xr = x + r * width;
#pragma unroll
    for (int j = 0; j < R::kKeep; ++j) {
        const int c = R::col(j);
#pragma unroll
        for (int e = 0; e < VEC; ++e) keep.v[j][e] = c < width ? to_f(row[c + e]) * scale : 0.f;
        if (c < width) R::put(xr + c, keep.v[j]);
    }
    R::beyond(width, [&](int i) { xr[i] = to_f(row[i]) * scale; });   // read again by this thread alone
    next_input<A, VEC, KEEP>(xb + r * ldxb, xr, next, keep, gain, width, eps, buf);
}

// ADD: x += y / rms(y) * w and xb = the next sublayer's input; otherwise xb = x / rms(x) * w for a listed row.
template <typename A, int VEC, int KEEP, bool ADD>
__global__ void __launch_bounds__(512) norm_kernel(float* x, A* xb, long ldxb, const float* y, const float* w, const float* next,
                                                   const int* rows, int width, float eps) {
    __shared__ float buf[32];
    typedef RowVecs<VEC, KEEP> R;
    R weight, gain, keep, sum;
    weight.load(w, width, 0.f);
    if (ADD) gain.load(next, width, 1.f);
    pdl_trigger();
    pdl_wait();
    const int out_row = blockIdx.x;
    const long r = rows ? rows[out_row] : out_row;
    float* xr = x + r * width;
    const float* src = ADD ? y + r * width : xr;
    keep.load(src, width, 0.f);
    if (ADD) sum.load(xr, width, 0.f);
    float ss = keep.squares();
    R::beyond(width, [&](int i) { ss = fmaf(src[i], src[i], ss); });
    const float rms = 1.0f / sqrtf(block_sum(ss, buf) / (float)width + eps);
    A* xo = xb + out_row * ldxb;
#pragma unroll
    for (int j = 0; j < R::kKeep; ++j) {
        const int c = R::col(j);
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            const float v = keep.v[j][e] * rms * weight.v[j][e];
            keep.v[j][e] = ADD ? sum.v[j][e] + v : v;
        }
        if (c < width) {
            if (ADD) R::put(xr + c, keep.v[j]);
            else R::put(xo + c, keep.v[j]);
        }
    }
    R::beyond(width, [&](int i) {
        const float v = src[i] * rms * w[i];
        if (ADD) xr[i] += v;
        else xo[i] = from_f<A>(v);
    });
    if (ADD) next_input<A, VEC, KEEP>(xo, xr, next, keep, gain, width, eps, buf);
}

template <typename A>
__global__ void __launch_bounds__(256) gated_norm_kernel(A* out, long ldout, const float* o, long ldo, const A* gate, long ldg,
                                                         const float* w, int heads, int V, int groups, int gate_first,
                                                         float eps) {
    __shared__ float buf[32];
    pdl_trigger();
    pdl_wait();
    const int grp = blockIdx.x, t = threadIdx.x;
    const long r = blockIdx.y;
    const int part = heads * V / groups, c0 = grp * part, V8 = pad8(V);
    const float* orow = o + r * ldo;
    const A* grow = gate + r * ldg;
    float ss = 0.f;
    for (int i = t; i < part; i += 256) {
        const int c = c0 + i, col = (c / V) * V8 + c % V;
        float v = orow[col];
        if (gate_first) v *= silu_f(to_f(grow[col]));
        ss = fmaf(v, v, ss);
    }
    const float rms = 1.0f / sqrtf(block_sum(ss, buf) / (float)part + eps);
    for (int i = t; i < part; i += 256) {
        const int c = c0 + i, h = c / V, v0 = c - h * V, col = h * V8 + v0;
        const float v = orow[col] * silu_f(to_f(grow[col])) * rms * (w ? w[c] : 1.f);
        out[r * ldout + col] = from_f<A>(v);
        if (v0 == V - 1)
            for (int z = V; z < V8; ++z) out[r * ldout + h * V8 + z] = from_f<A>(0.f);
    }
}

// The same with one group per head and the gate last: a warp per head.
template <typename A>
__global__ void __launch_bounds__(256) gated_norm_heads_kernel(A* out, long ldout, const float* o, long ldo, const A* gate, long ldg,
                                                               const float* w, int heads, int V, float eps) {
    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, V8 = pad8(V);
    if (h >= heads) return;
    const long r = blockIdx.y;
    const float* orow = o + r * ldo + h * V8;
    const A* grow = gate + r * ldg + h * V8;
    A* dst = out + r * ldout + h * V8;
    constexpr int kVec = 4;   // first 512 columns in registers
    float4 x[kVec];
    float ss = 0.f;
    auto add = [&](const float4& v) { ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss)))); };
#pragma unroll
    for (int j = 0; j < kVec; ++j) {   // columns V .. V8 are zero
        const int c = j * 128 + lane * 4;
        x[j] = c < V8 ? *reinterpret_cast<const float4*>(orow + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        add(x[j]);
    }
    for (int c = kVec * 128 + lane * 4; c < V8; c += 128) add(*reinterpret_cast<const float4*>(orow + c));
    const float rms = 1.0f / sqrtf(warp_sum(ss) / (float)V + eps);
    auto emit = [&](int c, const float4& v) {
        const float y[4] = {v.x, v.y, v.z, v.w};
        float z[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) z[e] = c + e < V ? y[e] * silu_f(to_f(grow[c + e])) * rms * (w ? w[(long)h * V + c + e] : 1.f) : 0.f;
        if constexpr (sizeof(A) == 2) *reinterpret_cast<uint2*>(dst + c) = make_uint2(pack_bf16(z[0], z[1]), pack_bf16(z[2], z[3]));
        else *reinterpret_cast<float4*>(dst + c) = make_float4(z[0], z[1], z[2], z[3]);
    };
#pragma unroll
    for (int j = 0; j < kVec; ++j)
        if (j * 128 + lane * 4 < V8) emit(j * 128 + lane * 4, x[j]);
    for (int c = kVec * 128 + lane * 4; c < V8; c += 128) emit(c, *reinterpret_cast<const float4*>(orow + c));
}

// Conv channel of a padded column (counted from the start of the convolved part), -1 for padding.
__device__ __forceinline__ int conv_channel(const ConvArgs& c, int col) {
    const int V8 = pad8(c.V), N8 = pad8(c.N), x_cols = c.heads * V8;
    if (col < x_cols) return col % V8 < c.V ? (col / V8) * c.V + col % V8 : -1;
    const int b = col - x_cols;   // k groups, then q groups
    return b % N8 < c.N ? c.heads * c.V + (b / N8) * c.N + b % N8 : -1;
}
__host__ __device__ __forceinline__ int conv_cols(const ConvArgs& c) { return c.heads * pad8(c.V) + 2 * c.groups * pad8(c.N); }

// Step size (or strength) and log decay of rows [t0, t1) of head h.
__device__ __forceinline__ void step_sizes(const ConvArgs& c, int h, int t0, int t1) {
    const float a = -expf(c.A_log[h]), b = c.dt_bias[h];
    for (int t = t0; t < t1; ++t) {
        const float dt = softplus_f(c.dt_raw[(long)t * c.ld_dt + h] + b);
        c.log_decay[(long)t * c.heads + h] = a * dt;
        c.weight[(long)t * c.heads + h] = c.beta_raw ? sigmoid_f(c.beta_raw[(long)t * c.ld_dt + h]) : dt;
    }
}

constexpr int kConvRows = 8;   // rows per block

template <typename A>
__global__ void __launch_bounds__(128) conv_silu_kernel(const ConvArgs c, const Rows r) {
    pdl_wait();
    const int channels = c.heads * c.V + 2 * c.groups * c.N, cols = conv_cols(c);
    const int col = blockIdx.x * 128 + threadIdx.x, t0 = blockIdx.y * kConvRows, t1 = min(r.T, t0 + kConvRows);
    if (col < cols) {
        const int ch = conv_channel(c, col);
        if (ch < 0) {
            for (int t = t0; t < t1; ++t) static_cast<A*>(c.out)[(long)t * c.ldo + col] = from_f<A>(0.f);
            return;
        }
        const A* u = static_cast<const A*>(c.u) + c.off + col;
        const float* ring = c.ring + (long)r.slot * c.taps * channels + ch;
        const float bias = c.bias ? c.bias[ch] : 0.f;
        for (int t = t0; t < t1; ++t) {
            float y = bias;
            for (int j = 0; j < c.taps; ++j) {
                const int s = t - (c.taps - 1) + j, p = r.pos0 + s;
                float v = 0.f;
                if (s >= 0) v = to_f(u[(long)s * c.ldu]);
                else if (p >= 0) v = ring[(long)(p % c.taps) * channels];
                y = fmaf(c.w[ch * c.taps + j], v, y);
            }
            static_cast<A*>(c.out)[(long)t * c.ldo + col] = from_f<A>(silu_f(y));
        }
    } else if (col < cols + c.heads) {
        step_sizes(c, col - cols, t0, t1);
    }
}

// bf16 prompts and few taps: a thread walks down 16 rows of eight columns (always of one head block) with the last inputs in
// registers.
constexpr int kConvWalk = 16;
template <int TAPS>
__global__ void __launch_bounds__(128) conv_walk_kernel(const ConvArgs c, const Rows r) {
    pdl_wait();
    const int channels = c.heads * c.V + 2 * c.groups * c.N, vecs = conv_cols(c) / 8;
    const int vec = blockIdx.x * 128 + threadIdx.x, t0 = blockIdx.y * kConvWalk, t1 = min(r.T, t0 + kConvWalk);
    if (vec >= vecs) {
        if (vec < vecs + c.heads) step_sizes(c, vec - vecs, t0, t1);
        return;
    }
    const bf16* u = static_cast<const bf16*>(c.u) + c.off + vec * 8;
    bf16* out = static_cast<bf16*>(c.out) + vec * 8;
    auto unpack = [](const uint4& v, float (&x)[8]) {
        const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            x[2 * i] = __uint_as_float(w[i] << 16);
            x[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u);
        }
    };
    float w[TAPS][8], bias[8], win[TAPS][8];   // win[i]: the input TAPS - 1 - i rows back
#pragma unroll
    for (int e = 0; e < 8; ++e) {
        const int ch = conv_channel(c, vec * 8 + e);   // padding columns: zero weights, zero output
        bias[e] = ch >= 0 && c.bias ? c.bias[ch] : 0.f;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) w[j][e] = ch >= 0 ? c.w[ch * TAPS + j] : 0.f;
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) {
            const int s = t0 - (TAPS - 1) + j, p = r.pos0 + s;
            float v = 0.f;
            if (s >= 0) v = to_f(u[(long)s * c.ldu + e]);
            else if (p >= 0 && ch >= 0) v = c.ring[((long)r.slot * TAPS + p % TAPS) * channels + ch];
            win[j][e] = v;
        }
    }
#pragma unroll 4
    for (int t = t0; t < t1; ++t) {
        unpack(*reinterpret_cast<const uint4*>(u + (long)t * c.ldu), win[TAPS - 1]);
        float y[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
            y[e] = bias[e];
#pragma unroll
            for (int j = 0; j < TAPS; ++j) y[e] = fmaf(w[j][e], win[j][e], y[e]);
            y[e] = __fdividef(y[e], 1.0f + __expf(-y[e]));
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j) win[j][e] = win[j + 1][e];
        }
        *reinterpret_cast<uint4*>(out + (long)t * c.ldo) =
            make_uint4(pack_bf16(y[0], y[1]), pack_bf16(y[2], y[3]), pack_bf16(y[4], y[5]), pack_bf16(y[6], y[7]));
    }
}
template <int TAPS>
cudaError_t conv_walk(const ConvArgs& c, const Rows& r, cudaStream_t st) {
    return launch_pdl(conv_walk_kernel<TAPS>, dim3((conv_cols(c) / 8 + c.heads + 127) / 128, (r.T + kConvWalk - 1) / kConvWalk), dim3(128), 0, st, c, r);
}

template <typename A>
__global__ void __launch_bounds__(128) conv_ring_kernel(const ConvArgs c, const Rows r) {
    pdl_wait();
    const int channels = c.heads * c.V + 2 * c.groups * c.N, col = blockIdx.x * 128 + threadIdx.x;
    const int ch = col < conv_cols(c) ? conv_channel(c, col) : -1;
    if (ch < 0) return;
    const A* u = static_cast<const A*>(c.u) + c.off + col;
    float* ring = c.ring + (long)r.slot * c.taps * channels + ch;
    for (int t = max(0, r.T - (c.taps - 1)); t < r.T; ++t) ring[(long)((r.pos0 + t) % c.taps) * channels] = to_f(u[(long)t * c.ldu]);
}

}  // namespace

namespace {

// threads of a row kernel: one access per thread, up to 512
int row_threads(int width, int vec) { return std::min(512, std::max(64, (width / vec + 31) / 32 * 32)); }

// Calls f<VEC, KEEP>() with the instance for this width.
template <typename F>
cudaError_t by_width(int width, F f) {
    if (width % 4 != 0) return f.template operator()<1, 4>();
    return width <= 2048 ? f.template operator()<4, 1>() : width <= 4096 ? f.template operator()<4, 2>() : f.template operator()<4, 4>();
}
template <typename A>
struct Embed {
    float* x; void* xb; long ldxb; const bf16* table; long ldt; const int* tokens; int T, width, vocab; float scale; const float* next;
    float eps; cudaStream_t st;
    template <int VEC, int KEEP>
    cudaError_t operator()() const {
        return launch_pdl(embed_kernel<A, VEC, KEEP>, dim3(T), dim3(row_threads(width, VEC)), 0, st, x, static_cast<A*>(xb), ldxb, table, ldt,
                          tokens, width, vocab, scale, next, eps);
    }
};
template <typename A, bool ADD>
struct Norm {
    float* x; void* xb; long ldxb; const float *y, *w, *next; const int* rows; int T, width; float eps; cudaStream_t st;
    template <int VEC, int KEEP>
    cudaError_t operator()() const {
        return launch_pdl(norm_kernel<A, VEC, KEEP, ADD>, dim3(T), dim3(row_threads(width, VEC)), 0, st, x, static_cast<A*>(xb), ldxb, y, w, next,
                          rows, width, eps);
    }
};

}  // namespace

cudaError_t embed(float* x, void* xb, long ldxb, const bf16* table, long ldt, const int* tokens, int T, int width, int vocab,
                  float scale, const float* next, float eps, int f32, cudaStream_t st) {
    count_launch(1);
    return f32 ? by_width(width, Embed<float>{x, xb, ldxb, table, ldt, tokens, T, width, vocab, scale, next, eps, st})
               : by_width(width, Embed<bf16>{x, xb, ldxb, table, ldt, tokens, T, width, vocab, scale, next, eps, st});
}

cudaError_t norm_add(float* x, void* xb, long ldxb, const float* y, const float* w, const float* next, int T, int width, float eps,
                     int f32, cudaStream_t st) {
    count_launch(1);
    return f32 ? by_width(width, Norm<float, true>{x, xb, ldxb, y, w, next, nullptr, T, width, eps, st})
               : by_width(width, Norm<bf16, true>{x, xb, ldxb, y, w, next, nullptr, T, width, eps, st});
}

cudaError_t norm_rows(void* xb, long ldxb, const float* x, const float* w, const int* rows, int T, int width, float eps, int f32,
                      cudaStream_t st) {
    count_launch(1);
    float* xm = const_cast<float*>(x);
    return f32 ? by_width(width, Norm<float, false>{xm, xb, ldxb, nullptr, w, nullptr, rows, T, width, eps, st})
               : by_width(width, Norm<bf16, false>{xm, xb, ldxb, nullptr, w, nullptr, rows, T, width, eps, st});
}

cudaError_t gated_norm(void* out, long ldout, const float* o, long ldo, const void* gate, long ldg, const float* w, int T,
                       int heads, int V, int groups, int gate_first, float eps, int f32, cudaStream_t st) {
    if (groups < 1 || (heads * V) % groups != 0) return cudaErrorInvalidValue;
    const dim3 grid(groups, T), block(256);
    count_launch(1);
    if (groups == heads && !gate_first) {
        const dim3 by_heads((heads + 7) / 8, T);
        return f32 ? launch_pdl(gated_norm_heads_kernel<float>, by_heads, block, 0, st, static_cast<float*>(out), ldout, o, ldo,
                                static_cast<const float*>(gate), ldg, w, heads, V, eps)
                   : launch_pdl(gated_norm_heads_kernel<bf16>, by_heads, block, 0, st, static_cast<bf16*>(out), ldout, o, ldo,
                                static_cast<const bf16*>(gate), ldg, w, heads, V, eps);
    }
    return f32 ? launch_pdl(gated_norm_kernel<float>, grid, block, 0, st, static_cast<float*>(out), ldout, o, ldo,
                            static_cast<const float*>(gate), ldg, w, heads, V, groups, gate_first, eps)
               : launch_pdl(gated_norm_kernel<bf16>, grid, block, 0, st, static_cast<bf16*>(out), ldout, o, ldo,
                            static_cast<const bf16*>(gate), ldg, w, heads, V, groups, gate_first, eps);
}

cudaError_t conv_silu(const ConvArgs& c, const Rows& r, int f32, cudaStream_t st) {
    const int n = conv_cols(c) + c.heads;
    const dim3 grid((n + 127) / 128, (r.T + kConvRows - 1) / kConvRows), block(128);
    count_launch(1);
    if (!f32 && r.T >= kConvWalk) {
        if (c.taps == 2) return conv_walk<2>(c, r, st);
        if (c.taps == 3) return conv_walk<3>(c, r, st);
        if (c.taps == 4) return conv_walk<4>(c, r, st);
    }
    return f32 ? launch_pdl(conv_silu_kernel<float>, grid, block, 0, st, c, r) : launch_pdl(conv_silu_kernel<bf16>, grid, block, 0, st, c, r);
}

cudaError_t conv_ring_store(const ConvArgs& c, const Rows& r, int f32, cudaStream_t st) {
    const dim3 grid((conv_cols(c) + 127) / 128), block(128);
    count_launch(1);
    return f32 ? launch_pdl(conv_ring_kernel<float>, grid, block, 0, st, c, r) : launch_pdl(conv_ring_kernel<bf16>, grid, block, 0, st, c, r);
}

}  // namespace lm
}  // namespace bw
