// Attention over a latent cache: a position is cached as one vector [latent (R) | rotated key part], shared by all heads;
// per head the unrotated key is W_uk c and the value W_uv c.  Softmax with a per-head sink in the denominator, a
// sigmoid gate per head on the output.
//   absorbed form (decode, short portions): the query is multiplied by W_uk once (latent_prep_kernel), after which all heads
//     attend to the cached rows themselves -- one pass over the cache for 16 heads at a time (latent_decode_kernel,
//     split over the context) -- and the weighted latent goes through W_uv (latent_out_kernel, which also merges the
//     splits, adds the sink and applies the gate).
//   expanded form (prompts): W_uk / W_uv are applied to the whole context with one matrix product, then flash attention
//     per head (latent_flash_kernel).
// Scores, softmax and sums are fp32.  In the bf16 kernels the absorbed query and the softmax weights enter the MMA as a
// high part plus a remainder.
#pragma once
#include "lm_device.cuh"
#include "lm_ops.h"

namespace bw {
namespace lm {

__device__ __forceinline__ float rot_elem(const float2* cs, int i, float self, float pair) {
    // element i of the rotated part: even i -> u cos - v sin (self = u, pair = v), odd i -> v cos + u sin
    const float2 w = cs[i >> 1];
    return (i & 1) ? self * w.x + pair * w.y : self * w.x - pair * w.y;
}

// ------------------------------------------------------------------------------------------ cache entries
template <typename A>
__device__ __forceinline__ void write_entry(const LatentArgs& a, const Rows& r, int row, float* buf) {
    const int slot = r.slot_of(row), pos = r.pos_of(row);
    const float* u = a.dkv + (long)row * a.ld32;
    float ss = 0.f;
    for (int i = threadIdx.x; i < a.R; i += blockDim.x) ss = fmaf(u[i], u[i], ss);
    const float rms = 1.0f / sqrtf(block_sum(ss, buf) / (float)a.R + a.eps);
    if (slot < 0 || pos >= a.max_seq) return;
    A* e = static_cast<A*>(a.cache) + ((long)slot * a.max_seq + pos) * a.ldc;
    const int R8 = pad8(a.R), rot8 = pad8(a.rot);
    const float2* cs = a.cs + (long)pos * (a.rot_dims / 2);
    for (int i = threadIdx.x; i < R8 + rot8; i += blockDim.x) {
        float v = 0.f;
        if (i < a.R) v = u[i] * rms * a.dkv_norm[i];
        else if (i >= R8 && i < R8 + a.rot) {
            const int d = i - R8;
            const float self = u[a.R + d];
            v = d < a.rot_dims ? rot_elem(cs, d, self, u[a.R + (d ^ 1)]) : self;
        }
        e[i] = from_f<A>(v);
    }
}
template <typename A>
__global__ void __launch_bounds__(128) latent_cache_kernel(const LatentArgs a, const Rows r) {
    __shared__ float buf[32];
    pdl_trigger();
    pdl_wait();
    write_entry<A>(a, r, blockIdx.x, buf);
}

// Rotates the queries' rotated part in place (expanded form).
__global__ void __launch_bounds__(128) latent_rotate_q_kernel(const LatentArgs a, const Rows r) {
    pdl_trigger();
    pdl_wait();
    const int half = a.rot_dims / 2, i = blockIdx.x * 128 + threadIdx.x, row = blockIdx.y;
    if (i >= a.heads * half) return;
    const int h = i / half, p = i - h * half;
    uint32_t* q = reinterpret_cast<uint32_t*>(static_cast<bf16*>(a.q) + (long)row * a.ldq + h * (pad8(a.dim) + pad8(a.rot)) + pad8(a.dim)) + p;
    const float2 w = a.cs[(long)r.pos_of(row) * half + p];
    const uint32_t v = *q;
    const float x = __uint_as_float(v << 16), y = __uint_as_float(v & 0xFFFF0000u);
    *q = pack_bf16(x * w.x - y * w.y, y * w.x + x * w.y);
}

// ------------------------------------------------------------------------------------------ absorbed form
constexpr int kPrepThreads = 256;

// Block (head, group of RB rows): q_abs = W_uk^T q and the rotated part.  One more block per row group writes the cache.
template <typename A, int RB>
__global__ void __launch_bounds__(kPrepThreads) latent_prep_kernel(const LatentArgs a, const Rows r) {
    extern __shared__ float sm[];
    const int h = blockIdx.x, row0 = blockIdx.y * RB, t = threadIdx.x;
    pdl_trigger();
    pdl_wait();
    if (h == a.heads) {
        for (int b = 0; b < RB; ++b)
            if (row0 + b < r.T) write_entry<A>(a, r, row0 + b, sm);
        return;
    }
    const int dim8 = pad8(a.dim), rot8 = pad8(a.rot), R8 = pad8(a.R), Dp = latent_dp(a.R, a.rot), nc = R8 / 8;
    float* qs = sm;                         // [RB][dim8 + rot8]
    float* red = qs + RB * (dim8 + rot8);   // [groups][RB][R8]
    for (int i = t; i < RB * (dim8 + rot8); i += kPrepThreads) {
        const int b = i / (dim8 + rot8), d = i - b * (dim8 + rot8);
        float v = 0.f;
        if (row0 + b < r.T) {
            const A* q = static_cast<const A*>(a.q) + (long)(row0 + b) * a.ldq + h * (dim8 + rot8);
            v = to_f(q[d]);
            const int e = d - dim8;
            if (e >= 0 && e < a.rot_dims) {
                const int p = min(r.pos_of(row0 + b), a.max_seq - 1);
                v = rot_elem(a.cs + (long)max(p, 0) * (a.rot_dims / 2), e, v, to_f(q[d ^ 1]));
            }
        }
        qs[i] = v;
    }
    __syncthreads();
    const int groups = max(1, kPrepThreads / nc), grp = t / nc;
    if (grp < groups || nc > kPrepThreads) {
        for (int c = nc > kPrepThreads ? t : t % nc; c < nc; c += nc > kPrepThreads ? kPrepThreads : nc) {
            float acc[RB][8] = {};
            const bf16* W = a.Wkv + (long)h * dim8 * a.ldw + c * 8;
#pragma unroll 8
            for (int d = nc > kPrepThreads ? 0 : grp; d < a.dim; d += groups) {
                const uint4 w = __ldg(reinterpret_cast<const uint4*>(W + (long)d * a.ldw));
                const uint32_t ww[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
                for (int b = 0; b < RB; ++b) {
                    const float q = qs[b * (dim8 + rot8) + d];
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        acc[b][2 * j] = fmaf(q, __uint_as_float(ww[j] << 16), acc[b][2 * j]);
                        acc[b][2 * j + 1] = fmaf(q, __uint_as_float(ww[j] & 0xFFFF0000u), acc[b][2 * j + 1]);
                    }
                }
            }
#pragma unroll
            for (int b = 0; b < RB; ++b) {
                float* o = red + ((long)(nc > kPrepThreads ? 0 : grp) * RB + b) * R8 + c * 8;
                *reinterpret_cast<float4*>(o) = make_float4(acc[b][0], acc[b][1], acc[b][2], acc[b][3]);
                *reinterpret_cast<float4*>(o + 4) = make_float4(acc[b][4], acc[b][5], acc[b][6], acc[b][7]);
            }
        }
    }
    __syncthreads();
    for (int i = t; i < RB * Dp; i += kPrepThreads) {
        const int b = i / Dp, d = i - b * Dp;
        if (row0 + b >= r.T) break;
        float v = 0.f;
        if (d < R8) {
            for (int g = 0; g < groups; ++g) v += red[((long)g * RB + b) * R8 + d];
        } else if (d < R8 + rot8) {
            v = qs[b * (dim8 + rot8) + dim8 + (d - R8)];
        }
        const long base = ((long)(row0 + b) * a.heads + h);
        if (sizeof(A) == 4) {
            static_cast<float*>(a.qabs)[base * Dp + d] = v;
        } else {
            bf16* o = static_cast<bf16*>(a.qabs) + base * 2 * Dp + d;
            const bf16 hi = __float2bfloat16_rn(v);
            o[0] = hi;
            o[Dp] = __float2bfloat16_rn(v - __bfloat162float(hi));
        }
    }
}

// One partial result per (row, head, split): R un-normalised outputs, then the running maximum and the sum.
__device__ __forceinline__ float* part_ptr(const LatentArgs& a, int row, int h, int split) {
    return a.part + (((long)row * a.heads + h) * a.splits + split) * (a.R + 2);
}

// Scalar kernel (32-bit mode; latent sizes the tensor-core kernel does not take): block (split, head, row).
constexpr int kScalarKeys = 32;
template <typename A>
__global__ void __launch_bounds__(256) latent_scalar_kernel(const LatentArgs a, const Rows r) {
    extern __shared__ float sm[];
    const int Dp = latent_dp(a.R, a.rot), R8 = pad8(a.R), rot8 = pad8(a.rot);
    float* q = sm;                        // [Dp]
    float* sc = q + Dp;                   // [kScalarKeys]
    const int t = threadIdx.x, warp = t >> 5, lane = t & 31;
    const int split = blockIdx.x, h = blockIdx.y, row = blockIdx.z;
    pdl_trigger();
    pdl_wait();
    const int slot = r.slot_of(row), len = min(r.pos_of(row) + 1, a.max_seq);
    float* out = part_ptr(a, row, h, split);
    const int tiles = (len + kScalarKeys - 1) / kScalarKeys, per = (tiles + a.splits - 1) / a.splits;
    const int k0 = min(split * per * kScalarKeys, len), k1 = min((split + 1) * per * kScalarKeys, len);
    if (slot < 0 || k0 >= k1) {
        if (t == 0) { out[a.R] = -INFINITY; out[a.R + 1] = 0.f; }
        return;
    }
    const long base = (long)row * a.heads + h;
    for (int i = t; i < Dp; i += 256)
        q[i] = sizeof(A) == 4 ? static_cast<const float*>(a.qabs)[base * Dp + i]
                              : to_f(static_cast<const bf16*>(a.qabs)[base * 2 * Dp + i]) + to_f(static_cast<const bf16*>(a.qabs)[(base * 2 + 1) * Dp + i]);
    constexpr int kCols = 8;              // latent columns per thread: 2048 at most
    float acc[kCols] = {};
    float m = -INFINITY, l = 0.f;
    const A* cache = static_cast<const A*>(a.cache) + (long)slot * a.max_seq * a.ldc;
    for (int kt = k0; kt < k1; kt += kScalarKeys) {
        const int n = min(kScalarKeys, k1 - kt);
        __syncthreads();
        for (int j = warp; j < n; j += 8) {
            const A* e = cache + (long)(kt + j) * a.ldc;
            float s = 0.f;
            for (int i = lane; i < R8 + rot8; i += 32) s = fmaf(q[i], to_f(e[i]), s);
            s = warp_sum(s);
            if (lane == 0) sc[j] = s * a.scale;
        }
        __syncthreads();
        float mn = m;
        for (int j = 0; j < n; ++j) mn = fmaxf(mn, sc[j]);
        const float alpha = expf(m - mn);
        l *= alpha;
#pragma unroll
        for (int c = 0; c < kCols; ++c) acc[c] *= alpha;
        for (int j = 0; j < n; ++j) {
            const float p = expf(sc[j] - mn);
            l += p;
            const A* e = cache + (long)(kt + j) * a.ldc;
#pragma unroll
            for (int c = 0; c < kCols; ++c)
                if (c * 256 + t < a.R) acc[c] = fmaf(p, to_f(e[c * 256 + t]), acc[c]);
        }
        m = mn;
    }
#pragma unroll
    for (int c = 0; c < kCols; ++c)
        if (c * 256 + t < a.R) out[c * 256 + t] = acc[c];
    if (t == 0) { out[a.R] = m; out[a.R + 1] = l; }
}

constexpr int kDecKeys = 64;
constexpr int kDecP = kDecKeys * 2 + 16;   // bytes of a row of softmax weights
struct DecodeSmem {
    int row, q_off, k_off, kbuf, p_off, f_off, total;
    __host__ __device__ DecodeSmem(int R, int rot, int nbuf) {
        row = latent_dp(R, rot) * 2 + 16;
        q_off = 0;
        k_off = 2 * 16 * row;
        kbuf = kDecKeys * row;
        p_off = k_off + nbuf * kbuf;
        f_off = p_off + 2 * 16 * kDecP;
        total = f_off + 2 * 8 * 16 * 4;
    }
};

// Block (split, 16 heads, row); 8 warps: warp w scores keys 8w .. 8w+7 of a 64-key tile and accumulates latent columns
// [w * NT * 8, (w + 1) * NT * 8).
template <int NT>
__global__ void __launch_bounds__(256) latent_decode_kernel(const LatentArgs a, const Rows r, int nbuf) {
    extern __shared__ __align__(16) unsigned char smem[];
    const DecodeSmem L(a.R, a.rot, nbuf);
    const int Dp = latent_dp(a.R, a.rot), R8 = pad8(a.R), D8 = R8 + pad8(a.rot);
    const int t = threadIdx.x, warp = t >> 5, lane = t & 31, g = lane >> 2, q4 = lane & 3;
    const int split = blockIdx.x, h0 = blockIdx.y * 16, row = blockIdx.z;
    const uint32_t sb = smem_u32(smem);
    float* redm = reinterpret_cast<float*>(smem + L.f_off);   // [8][16]
    float* redl = redm + 8 * 16;
    pdl_trigger();
    pdl_wait();
    const int slot = r.slot_of(row), len = min(r.pos_of(row) + 1, a.max_seq);
    const int tiles = (len + kDecKeys - 1) / kDecKeys, per = (tiles + a.splits - 1) / a.splits;
    const int t0 = split * per, t1 = min(tiles, t0 + per);
    if (slot < 0 || t0 >= t1) {
        if (t < 16 && h0 + t < a.heads) {
            float* out = part_ptr(a, row, h0 + t, split);
            out[a.R] = -INFINITY;
            out[a.R + 1] = 0.f;
        }
        return;
    }
    const bf16* cache = static_cast<const bf16*>(a.cache) + (long)slot * a.max_seq * a.ldc;
    const int nc = Dp / 8;
    auto issue = [&](int tile, int buf) {
        for (int i = t; i < kDecKeys * nc; i += 256) {
            const int k = i / nc, c = (i - k * nc) * 8, key = tile * kDecKeys + k;
            const bool ok = key < len && c < D8;
            cp_async16z(sb + L.k_off + buf * L.kbuf + k * L.row + c * 2, ok ? cache + (long)key * a.ldc + c : cache, ok);
        }
        cp_async_commit();
    };
    for (int i = t; i < 2 * 16 * nc; i += 256) {
        const int part = i / (16 * nc), rem = i - part * 16 * nc, hh = rem / nc, c = (rem - hh * nc) * 8;
        const bool ok = h0 + hh < a.heads;
        const bf16* q = static_cast<const bf16*>(a.qabs);
        cp_async16z(sb + L.q_off + (part * 16 + hh) * L.row + c * 2, ok ? q + (((long)row * a.heads + h0 + hh) * 2 + part) * Dp + c : q, ok);
    }
    issue(t0, 0);
    float O[NT][4] = {};
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
    for (int tile = t0; tile < t1; ++tile) {
        const int buf = nbuf == 2 ? (tile - t0) & 1 : 0;
        const uint32_t kb = sb + L.k_off + buf * L.kbuf;
        cp_async_wait<0>();
        __syncthreads();
        if (nbuf == 2 && tile + 1 < t1) issue(tile + 1, buf ^ 1);
        float s[4] = {}, sl[4] = {};
        for (int k0 = 0; k0 < Dp; k0 += 16) {
            uint32_t ah[4], al[4], b[2];
            const uint32_t qa = sb + L.q_off + (lane & 15) * L.row + (k0 + (lane >> 4) * 8) * 2;
            ldsm4(qa, ah);
            ldsm4(qa + 16 * L.row, al);
            ldsm2(kb + (8 * warp + (lane & 7)) * L.row + (k0 + ((lane >> 3) & 1) * 8) * 2, b);
            mma_bf16(s, ah[0], ah[1], ah[2], ah[3], b[0], b[1]);
            mma_bf16(sl, al[0], al[1], al[2], al[3], b[0], b[1]);
        }
        const int key = tile * kDecKeys + 8 * warp + 2 * q4;
#pragma unroll
        for (int i = 0; i < 4; ++i) s[i] = key + (i & 1) < len ? (s[i] + sl[i]) * a.scale : -INFINITY;
        float x0 = fmaxf(s[0], s[1]), x1 = fmaxf(s[2], s[3]);
#pragma unroll
        for (int o = 1; o <= 2; o <<= 1) {
            x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, o));
            x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, o));
        }
        if (q4 == 0) { redm[warp * 16 + g] = x0; redm[warp * 16 + g + 8] = x1; }
        __syncthreads();
        float n0 = m0, n1 = m1;
#pragma unroll
        for (int w = 0; w < 8; ++w) { n0 = fmaxf(n0, redm[w * 16 + g]); n1 = fmaxf(n1, redm[w * 16 + g + 8]); }
        const float al0 = expf(m0 - n0), al1 = expf(m1 - n1);   // the tile's first key is always visible: n is finite
        m0 = n0;
        m1 = n1;
        const float p0 = expf(s[0] - n0), p1 = expf(s[1] - n0), p2 = expf(s[2] - n1), p3 = expf(s[3] - n1);
        uint32_t hi, lo;
        unsigned char* pd = smem + L.p_off + g * kDecP + (8 * warp + 2 * q4) * 2;
        split_bf16(p0, p1, hi, lo);
        *reinterpret_cast<uint32_t*>(pd) = hi;
        *reinterpret_cast<uint32_t*>(pd + 16 * kDecP) = lo;
        split_bf16(p2, p3, hi, lo);
        *reinterpret_cast<uint32_t*>(pd + 8 * kDecP) = hi;
        *reinterpret_cast<uint32_t*>(pd + 24 * kDecP) = lo;
        float y0 = p0 + p1, y1 = p2 + p3;
#pragma unroll
        for (int o = 1; o <= 2; o <<= 1) {
            y0 += __shfl_xor_sync(0xffffffffu, y0, o);
            y1 += __shfl_xor_sync(0xffffffffu, y1, o);
        }
        if (q4 == 0) { redl[warp * 16 + g] = y0; redl[warp * 16 + g + 8] = y1; }
        __syncthreads();
        l0 *= al0;
        l1 *= al1;
#pragma unroll
        for (int w = 0; w < 8; ++w) { l0 += redl[w * 16 + g]; l1 += redl[w * 16 + g + 8]; }
#pragma unroll
        for (int j = 0; j < NT; ++j) { O[j][0] *= al0; O[j][1] *= al0; O[j][2] *= al1; O[j][3] *= al1; }
#pragma unroll
        for (int k0 = 0; k0 < kDecKeys; k0 += 16) {
            uint32_t ph[4], pl[4];
            const uint32_t pa = sb + L.p_off + (lane & 15) * kDecP + (k0 + (lane >> 4) * 8) * 2;
            ldsm4(pa, ph);
            ldsm4(pa + 16 * kDecP, pl);
#pragma unroll
            for (int j = 0; j < NT; j += 2) {
                const int col = (warp * NT + j) * 8;
                if (col < R8) {
                    uint32_t v[4];
                    ldsm4t(kb + (k0 + (lane & 15)) * L.row + (col + (lane >> 4) * 8) * 2, v);
                    mma_bf16(O[j], ph[0], ph[1], ph[2], ph[3], v[0], v[1]);
                    mma_bf16(O[j + 1], ph[0], ph[1], ph[2], ph[3], v[2], v[3]);
                    mma_bf16(O[j], pl[0], pl[1], pl[2], pl[3], v[0], v[1]);
                    mma_bf16(O[j + 1], pl[0], pl[1], pl[2], pl[3], v[2], v[3]);
                }
            }
        }
        if (nbuf == 1) {
            __syncthreads();
            if (tile + 1 < t1) issue(tile + 1, 0);
        }
    }
#pragma unroll
    for (int p = 0; p < 2; ++p) {
        const int h = h0 + g + 8 * p;
        if (h >= a.heads) continue;
        float* out = part_ptr(a, row, h, split);
#pragma unroll
        for (int j = 0; j < NT; ++j) {
            const int col = (warp * NT + j) * 8 + 2 * q4;
            if (col < a.R) out[col] = O[j][2 * p];
            if (col + 1 < a.R) out[col + 1] = O[j][2 * p + 1];
        }
        if (warp == 0 && q4 == 0) {
            out[a.R] = p ? m1 : m0;
            out[a.R + 1] = p ? l1 : l0;
        }
    }
}

// Block (head, group of RB rows): merges the splits, adds the sink to the denominator, applies W_uv and the gate.
template <typename A, int RB>
__global__ void __launch_bounds__(256) latent_out_kernel(const LatentArgs a, const Rows r) {
    extern __shared__ float sm[];
    const int R8 = pad8(a.R), dim8 = pad8(a.dim), V8 = pad8(a.V);
    float* lat = sm;                     // [RB][R8]
    float* wsp = lat + RB * R8;          // [RB][splits] weights of the splits
    const int h = blockIdx.x, row0 = blockIdx.y * RB, t = threadIdx.x, warp = t >> 5, lane = t & 31;
    pdl_trigger();
    pdl_wait();
    if (warp < RB && row0 + warp < r.T) {
        const int row = row0 + warp;
        const float sink = a.sink[h];
        float m = sink;
        for (int s = lane; s < a.splits; s += 32) m = fmaxf(m, part_ptr(a, row, h, s)[a.R]);
        m = warp_max(m);
        float l = 0.f;
        for (int s = lane; s < a.splits; s += 32) {
            const float* p = part_ptr(a, row, h, s);
            const float w = p[a.R + 1] > 0.f ? expf(p[a.R] - m) : 0.f;
            wsp[warp * a.splits + s] = w;
            l += w > 0.f ? w * p[a.R + 1] : 0.f;
        }
        l = warp_sum(l) + expf(sink - m);
        __syncwarp();
        for (int s = lane; s < a.splits; s += 32) wsp[warp * a.splits + s] /= l;
    }
    __syncthreads();
    for (int i = t; i < RB * R8; i += 256) {
        const int b = i / R8, c = i - b * R8;
        float v = 0.f;
        if (row0 + b < r.T && c < a.R)
            for (int s = 0; s < a.splits; ++s) {
                const float w = wsp[b * a.splits + s];
                if (w > 0.f) v = fmaf(w, part_ptr(a, row0 + b, h, s)[c], v);
            }
        lat[i] = v;
    }
    __syncthreads();
    float gate[RB];
#pragma unroll
    for (int b = 0; b < RB; ++b) gate[b] = row0 + b < r.T ? sigmoid_f(a.gate[(long)(row0 + b) * a.ld32 + h]) : 0.f;
    const bf16* W = a.Wkv + ((long)a.heads * dim8 + (long)h * V8) * a.ldw;
#pragma unroll 2
    for (int v = warp; v < V8; v += 8) {
        float acc[RB] = {};
        if (v < a.V) {
#pragma unroll 2
            for (int c = lane * 8; c < R8; c += 256) {
                const uint4 w = __ldg(reinterpret_cast<const uint4*>(W + (long)v * a.ldw + c));
                const uint32_t ww[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
                for (int b = 0; b < RB; ++b) {
                    const float4 x0 = *reinterpret_cast<const float4*>(lat + b * R8 + c);
                    const float4 x1 = *reinterpret_cast<const float4*>(lat + b * R8 + c + 4);
                    acc[b] = fmaf(x0.x, __uint_as_float(ww[0] << 16), acc[b]);
                    acc[b] = fmaf(x0.y, __uint_as_float(ww[0] & 0xFFFF0000u), acc[b]);
                    acc[b] = fmaf(x0.z, __uint_as_float(ww[1] << 16), acc[b]);
                    acc[b] = fmaf(x0.w, __uint_as_float(ww[1] & 0xFFFF0000u), acc[b]);
                    acc[b] = fmaf(x1.x, __uint_as_float(ww[2] << 16), acc[b]);
                    acc[b] = fmaf(x1.y, __uint_as_float(ww[2] & 0xFFFF0000u), acc[b]);
                    acc[b] = fmaf(x1.z, __uint_as_float(ww[3] << 16), acc[b]);
                    acc[b] = fmaf(x1.w, __uint_as_float(ww[3] & 0xFFFF0000u), acc[b]);
                }
            }
        }
#pragma unroll
        for (int b = 0; b < RB; ++b) {
            const float s = warp_sum(acc[b]);
            if (lane == 0 && row0 + b < r.T)
                static_cast<A*>(a.out)[(long)(row0 + b) * a.ldout + h * V8 + v] = from_f<A>(s * gate[b]);
        }
    }
}

// ------------------------------------------------------------------------------------------ expanded form
constexpr int kFlashQ = 128, kFlashK = 64;
struct FlashSmem {
    int row, vrow, k_off, kbuf, total;
    __host__ __device__ FlashSmem(int D, int VT) {
        row = D * 2 + 16;
        vrow = VT * 16 + 16;
        k_off = kFlashQ * row;
        kbuf = kFlashK * (row + vrow);
        total = k_off + 2 * kbuf;
    }
};

// Block (128 query rows, head, slice of VT * 8 value columns); warp w has rows 16 w .. 16 w + 15.
template <int VT>
__global__ void __launch_bounds__(256, 1) latent_flash_kernel(const LatentArgs a, const Rows r) {
    extern __shared__ __align__(16) unsigned char smem[];
    const int dim8 = pad8(a.dim), rot8 = pad8(a.rot), D8 = dim8 + rot8, D = pad16(D8), V8 = pad8(a.V), R8 = pad8(a.R);
    const FlashSmem L(D, VT);
    const int t = threadIdx.x, warp = t >> 5, lane = t & 31, g = lane >> 2, q4 = lane & 3;
    const int q0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * kFlashQ, h = blockIdx.y, v0 = blockIdx.z * VT * 8;
    const uint32_t sb = smem_u32(smem);
    const bf16* kv = static_cast<const bf16*>(a.kv);
    const long ldkv = (long)a.heads * (dim8 + V8);
    const bf16* kr = static_cast<const bf16*>(a.cache) + (long)r.slot * a.max_seq * a.ldc + R8;
    const int last = min(r.T, q0 + kFlashQ) - 1;           // last real query row of the block
    const int nkeys = r.pos0 + last + 1, tiles = (nkeys + kFlashK - 1) / kFlashK;
    pdl_wait();
    auto issue = [&](int tile, int buf) {
        const uint32_t kb = sb + L.k_off + buf * L.kbuf, vb = kb + kFlashK * L.row;
        const int nc = D / 8;
        for (int i = t; i < kFlashK * nc; i += 256) {
            const int k = i / nc, c = (i - k * nc) * 8, key = tile * kFlashK + k;
            const bool ok = key < nkeys && c < D8;
            const bf16* src = c < dim8 ? kv + (long)key * ldkv + h * dim8 + c : kr + (long)key * a.ldc + (c - dim8);
            cp_async16z(kb + k * L.row + c * 2, ok ? src : kv, ok);
        }
        for (int i = t; i < kFlashK * VT; i += 256) {
            const int k = i / VT, c = (i - k * VT) * 8, key = tile * kFlashK + k;
            const bool ok = key < nkeys && v0 + c < V8;
            cp_async16z(vb + k * L.vrow + c * 2, ok ? kv + (long)key * ldkv + a.heads * dim8 + h * V8 + v0 + c : kv, ok);
        }
        cp_async_commit();
    };
    {
        const int nc = D / 8;
        for (int i = t; i < kFlashQ * nc; i += 256) {
            const int q = i / nc, c = (i - q * nc) * 8;
            const bool ok = q0 + q < r.T && c < D8;
            const bf16* src = static_cast<const bf16*>(a.q);
            cp_async16z(sb + q * L.row + c * 2, ok ? src + (long)(q0 + q) * a.ldq + h * D8 + c : src, ok);
        }
    }
    issue(0, 0);
    float O[VT][4] = {};
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
    const int wrow = q0 + 16 * warp;                       // first query row of the warp
    const float sl2 = a.scale * 1.4426950408889634f;       // softmax in base 2
    for (int tile = 0; tile < tiles; ++tile) {
        const int buf = tile & 1;
        const uint32_t kb = sb + L.k_off + buf * L.kbuf, vb = kb + kFlashK * L.row;
        cp_async_wait<0>();
        __syncthreads();
        if (tile + 1 < tiles) issue(tile + 1, buf ^ 1);
        if (tile * kFlashK > r.pos0 + wrow + 15) continue;  // nothing of this tile is visible to the warp
        float s[8][4] = {};
        for (int k0 = 0; k0 < D; k0 += 16) {
            uint32_t fa[4];
            ldsm4(sb + (16 * warp + (lane & 15)) * L.row + (k0 + (lane >> 4) * 8) * 2, fa);
#pragma unroll
            for (int jj = 0; jj < 4; ++jj) {
                uint32_t fb[4];
                ldsm4(kb + (16 * jj + (lane & 7) + (lane >> 4) * 8) * L.row + (k0 + ((lane >> 3) & 1) * 8) * 2, fb);
                mma_bf16(s[2 * jj], fa[0], fa[1], fa[2], fa[3], fb[0], fb[1]);
                mma_bf16(s[2 * jj + 1], fa[0], fa[1], fa[2], fa[3], fb[2], fb[3]);
            }
        }
        const bool edge = tile * kFlashK + kFlashK - 1 > r.pos0 + wrow;
#pragma unroll
        for (int p = 0; p < 2; ++p) {
            const int pos = r.pos0 + wrow + g + 8 * p;
            float mx = m[p];
#pragma unroll
            for (int j = 0; j < 8; ++j)
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    float& x = s[j][2 * p + i];
                    x *= sl2;
                    if (edge && tile * kFlashK + 8 * j + 2 * q4 + i > pos) x = -INFINITY;
                    mx = fmaxf(mx, x);
                }
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
            const float base = mx == -INFINITY ? 0.f : mx, alpha = exp2f(m[p] - base);
            m[p] = mx;
            float sum = 0.f;
#pragma unroll
            for (int j = 0; j < 8; ++j)
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    float& x = s[j][2 * p + i];
                    x = exp2f(x - base);
                    sum += x;
                }
            l[p] = l[p] * alpha + sum;
#pragma unroll
            for (int j = 0; j < VT; ++j) { O[j][2 * p] *= alpha; O[j][2 * p + 1] *= alpha; }
        }
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {   // 16 keys: the score fragments are the A operand
            uint32_t ph[4], pl[4];
            split_bf16(s[2 * kk][0], s[2 * kk][1], ph[0], pl[0]);
            split_bf16(s[2 * kk][2], s[2 * kk][3], ph[1], pl[1]);
            split_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1], ph[2], pl[2]);
            split_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3], ph[3], pl[3]);
#pragma unroll
            for (int j = 0; j < VT; j += 2) {
                uint32_t v[4];
                ldsm4t(vb + (16 * kk + (lane & 15)) * L.vrow + (8 * j + (lane >> 4) * 8) * 2, v);
                mma_bf16(O[j], ph[0], ph[1], ph[2], ph[3], v[0], v[1]);
                mma_bf16(O[j + 1], ph[0], ph[1], ph[2], ph[3], v[2], v[3]);
                mma_bf16(O[j], pl[0], pl[1], pl[2], pl[3], v[0], v[1]);
                mma_bf16(O[j + 1], pl[0], pl[1], pl[2], pl[3], v[2], v[3]);
            }
        }
    }
    const float sink = a.sink[h] * 1.4426950408889634f;
#pragma unroll
    for (int p = 0; p < 2; ++p) {
        const int q = wrow + g + 8 * p;
        float tot = l[p];
        tot += __shfl_xor_sync(0xffffffffu, tot, 1);
        tot += __shfl_xor_sync(0xffffffffu, tot, 2);
        if (q >= r.T) continue;
        const float mm = fmaxf(m[p], sink), sc = exp2f(m[p] - mm);
        const float f = sc / (tot * sc + exp2f(sink - mm)) * sigmoid_f(a.gate[(long)q * a.ld32 + h]);
        bf16* out = static_cast<bf16*>(a.out) + (long)q * a.ldout + h * V8 + v0;
#pragma unroll
        for (int j = 0; j < VT; ++j) {
            const int col = 8 * j + 2 * q4;
            if (v0 + col < V8) *reinterpret_cast<uint32_t*>(out + col) = pack_bf16(O[j][2 * p] * f, O[j][2 * p + 1] * f);
        }
    }
}

}  // namespace lm
}  // namespace bw
