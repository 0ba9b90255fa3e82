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

// Block (head, COLS latent columns; RB rows): q_abs = W_uk^T q, and from the first column block the rotated part.  RB more
// blocks per row group write the cache entries.  COLS / 8 threads cover the columns, the others split the query
// dimensions; the first weights are fetched before the kernel waits for its predecessor.
template <typename A, int RB, int COLS>
__global__ void __launch_bounds__(kPrepThreads) latent_prep_kernel(const LatentArgs a, const Rows r) {
    extern __shared__ __align__(16) float sm[];
    const int dim8 = pad8(a.dim), rot8 = pad8(a.rot), R8 = pad8(a.R), Dp = latent_dp(a.R, a.rot);
    const int cblocks = (R8 + COLS - 1) / COLS, t = threadIdx.x;
    const int h = blockIdx.x / cblocks, cb = blockIdx.x - h * cblocks, row0 = blockIdx.y * RB;
    pdl_trigger();
    if (h >= a.heads) {
        pdl_wait();
        const int row = row0 + (int)blockIdx.x - a.heads * cblocks;
        if (row < r.T) write_entry<A>(a, r, row, sm);
        return;
    }
    constexpr int TC = COLS / 8, GR = kPrepThreads / TC;   // threads across the columns, groups over the dimensions
    constexpr int kPre = RB > 1 ? 8 : 4;
    const int col = cb * COLS + (t % TC) * 8, grp = t / TC;
    const bf16* W = a.Wkv + (long)h * dim8 * a.ldw + col;
    uint4 pre[kPre];
#pragma unroll
    for (int i = 0; i < kPre; ++i)
        pre[i] = col < R8 && grp + GR * i < a.dim ? __ldg(reinterpret_cast<const uint4*>(W + (long)(grp + GR * i) * a.ldw)) : make_uint4(0, 0, 0, 0);
    pdl_wait();
    float* qs = sm;                                   // [dim8 + rot8][RB]
    float* red = qs + RB * (dim8 + rot8);             // [GR][RB][COLS]
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
        qs[d * RB + b] = v;
    }
    __syncthreads();
    float acc[RB][8] = {};
    auto add = [&](const uint4& w, int d) {
        const uint32_t ww[4] = {w.x, w.y, w.z, w.w};
        float q[RB];
        if (RB == 4) *reinterpret_cast<float4*>(q) = *reinterpret_cast<const float4*>(qs + d * RB);
        else
#pragma unroll
            for (int b = 0; b < RB; ++b) q[b] = qs[d * RB + b];
#pragma unroll
        for (int b = 0; b < RB; ++b)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                acc[b][2 * j] = fmaf(q[b], __uint_as_float(ww[j] << 16), acc[b][2 * j]);
                acc[b][2 * j + 1] = fmaf(q[b], __uint_as_float(ww[j] & 0xFFFF0000u), acc[b][2 * j + 1]);
            }
    };
#pragma unroll
    for (int i = 0; i < kPre; ++i)
        if (grp + GR * i < a.dim) add(pre[i], grp + GR * i);
    if (col < R8)
#pragma unroll 4
        for (int d = grp + GR * kPre; d < a.dim; d += GR) add(__ldg(reinterpret_cast<const uint4*>(W + (long)d * a.ldw)), d);
#pragma unroll
    for (int b = 0; b < RB; ++b) {
        float* o = red + (grp * RB + b) * COLS + (t % TC) * 8;
        *reinterpret_cast<float4*>(o) = make_float4(acc[b][0], acc[b][1], acc[b][2], acc[b][3]);
        *reinterpret_cast<float4*>(o + 4) = make_float4(acc[b][4], acc[b][5], acc[b][6], acc[b][7]);
    }
    __syncthreads();
    auto put = [&](int b, int d, float v) {
        const long base = ((long)(row0 + b) * a.heads + h);
        if (sizeof(A) == 4) {
            static_cast<float*>(a.qabs)[base * Dp + d] = v;
        } else {
            bf16* o = static_cast<bf16*>(a.qabs) + base * 2 * Dp + d;
            const bf16 hi = __float2bfloat16_rn(v);
            o[0] = hi;
            o[Dp] = __float2bfloat16_rn(v - __bfloat162float(hi));
        }
    };
    for (int i = t; i < RB * COLS; i += kPrepThreads) {
        const int b = i / COLS, c = i % COLS;
        if (row0 + b >= r.T || cb * COLS + c >= R8) continue;
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < GR; ++w) v += red[(w * RB + b) * COLS + c];
        put(b, cb * COLS + c, v);
    }
    if (cb == 0)
        for (int i = t; i < RB * (Dp - R8); i += kPrepThreads) {
            const int b = i / (Dp - R8), e = i - b * (Dp - R8);
            if (row0 + b < r.T) put(b, R8 + e, e < rot8 ? qs[(dim8 + e) * RB + b] : 0.f);
        }
}

// One partial result per (row, head, split): pad8(R) un-normalised outputs, then the running maximum and the sum.
__device__ __forceinline__ float* part_ptr(const LatentArgs& a, int row, int h, int split) {
    return a.part + (((long)row * a.heads + h) * a.splits + split) * (pad8(a.R) + kPartStats);
}
// Splits of a context of `len` positions that hold any (tiles of `keys` are dealt out in runs of equal length).
__device__ __forceinline__ int used_splits(int len, int keys, int splits) {
    const int tiles = (len + keys - 1) / keys, per = (tiles + splits - 1) / splits;
    return (tiles + per - 1) / per;
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
    float* stats = out + R8;
    const int tiles = (len + kScalarKeys - 1) / kScalarKeys, per = (tiles + a.splits - 1) / a.splits;
    const int k0 = min(split * per * kScalarKeys, len), k1 = min((split + 1) * per * kScalarKeys, len);
    if (slot < 0 || k0 >= k1) return;   // the merge reads the splits that hold positions
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
                if (c * 256 + t < R8) acc[c] = fmaf(p, to_f(e[c * 256 + t]), acc[c]);
        }
        m = mn;
    }
#pragma unroll
    for (int c = 0; c < kCols; ++c)
        if (c * 256 + t < R8) out[c * 256 + t] = acc[c];
    if (t == 0) { stats[0] = m; stats[1] = l; }
}

constexpr int kDecKeys = 32;               // keys per tile of a warp group
constexpr int kDecThreads = 512;           // two groups of eight warps
constexpr int kDecSteps = 5;               // 16-wide query steps a warp holds: padded query size up to 640
constexpr int kDecP = kDecKeys * 2 + 16;   // bytes of a row of softmax weights
constexpr int kDecS = kDecKeys + 4;        // floats of a row of partial scores
struct DecodeSmem {                        // per group: two key tiles, softmax weights, partial scores, rescale factors
    int row, kbuf, p_off, s_off, f_off, bar_off, group, total;
    __host__ __device__ DecodeSmem(int R, int rot) {
        row = latent_dp(R, rot) * 2 + 16;
        kbuf = kDecKeys * row;
        p_off = 2 * kbuf;
        s_off = p_off + 2 * 16 * kDecP;
        f_off = s_off + 8 * 16 * kDecS * 4;
        bar_off = f_off + 2 * 16 * 4;
        group = bar_off + 16;
        total = 2 * group;
    }
};
__device__ __forceinline__ void group_sync(int group) {
    if (group) asm volatile("bar.sync 2, 256;" ::: "memory");
    else asm volatile("bar.sync 1, 256;" ::: "memory");
}

// Block (split, 16 heads, row): the tiles of the split alternate between two warp groups that run independently, so that
// one group's products overlap the other's softmax; their results are merged at the end.  Inside a group a warp holds every
// eighth 16-wide step of the queries in registers and multiplies it with all keys of the tile; the partial scores meet
// in shared memory, where 16 neighbouring threads own one head's row.  Output: a warp accumulates latent columns
// [w * NT * 8, (w + 1) * NT * 8).
template <int NT>
__global__ void __launch_bounds__(kDecThreads) latent_decode_kernel(const LatentArgs a, const Rows r, int* status) {
    extern __shared__ __align__(16) unsigned char smem_all[];
    const DecodeSmem L(a.R, a.rot);
    const int Dp = latent_dp(a.R, a.rot), R8 = pad8(a.R), D8 = R8 + pad8(a.rot);
    const int group = threadIdx.x >> 8, t = threadIdx.x & 255, warp = t >> 5, lane = t & 31, g = lane >> 2, q4 = lane & 3;
    const int split = blockIdx.x, h0 = blockIdx.y * 16, row = blockIdx.z;
    unsigned char* smem = smem_all + group * L.group;
    const uint32_t sb = smem_u32(smem);
    float* part = reinterpret_cast<float*>(smem + L.s_off);    // [8][16][kDecS]
    float* alphas = reinterpret_cast<float*>(smem + L.f_off);  // [2][16]
    pdl_trigger();
    pdl_wait();
    const int slot = r.slot_of(row), len = min(r.pos_of(row) + 1, a.max_seq);
    const int tiles = (len + kDecKeys - 1) / kDecKeys, per = (tiles + a.splits - 1) / a.splits;
    const int t0 = split * per, t1 = min(tiles, t0 + per);
    if (slot < 0 || t0 >= t1) return;   // the merge reads the splits that hold positions
    const bf16* cache = static_cast<const bf16*>(a.cache) + (long)slot * a.max_seq * a.ldc;
    // rows past the sequence's end keep what the buffer held before (zeros or earlier keys): their weights are zero
    zero_smem(smem, 2 * L.kbuf, t, 256);
    if (t == 0) {
        mbar_init(sb + L.bar_off, 1);
        mbar_init(sb + L.bar_off + 8, 1);
        mbar_fence_init();
    }
    fence_proxy_async();
    group_sync(group);
    auto issue = [&](int tile, int buf) {   // one row per lane of the group's first warp
        const uint32_t bar = sb + L.bar_off + 8 * buf;
        const int key = tile * kDecKeys + lane;
        if (lane == 0) mbar_expect_tx(bar, min(kDecKeys, len - tile * kDecKeys) * D8 * 2);
        __syncwarp();
        if (key < len) bulk_row(sb + buf * L.kbuf + lane * L.row, cache + (long)key * a.ldc, D8 * 2, bar);
    };
    int tile = t0 + group;
    if (tile < t1 && warp == 0) issue(tile, 0);
    uint32_t qh[kDecSteps][4], ql[kDecSteps][4];   // query fragments: high parts, remainders
    {
        const long stride = 2L * Dp;               // bf16 per head: high parts, then remainders
        const uint32_t* q0 = reinterpret_cast<const uint32_t*>(static_cast<const bf16*>(a.qabs) + ((long)row * a.heads + h0 + g) * stride) + q4;
        const uint32_t* q1 = q0 + 8 * (stride / 2);
        const bool v0 = h0 + g < a.heads, v1 = h0 + g + 8 < a.heads;
#pragma unroll
        for (int i = 0; i < kDecSteps; ++i) {
            const int k = (warp + 8 * i) * 8;      // in 32-bit words
            const bool in = 2 * k < Dp;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                qh[i][2 * e] = in && v0 ? q0[k + 4 * e] : 0u;
                qh[i][2 * e + 1] = in && v1 ? q1[k + 4 * e] : 0u;
                ql[i][2 * e] = in && v0 ? q0[Dp / 2 + k + 4 * e] : 0u;
                ql[i][2 * e + 1] = in && v1 ? q1[Dp / 2 + k + 4 * e] : 0u;
            }
        }
    }
    float O[NT][4] = {};
    const int srow = t >> 4, skey = (t & 15) * 2;   // this thread's head row and keys in the softmax
    float m = -INFINITY, l = 0.f;
    CopyWait copied{status};
    uint32_t phases = 0;
    for (int buf = 0; tile < t1; tile += 2, buf ^= 1) {
        const uint32_t kb = sb + buf * L.kbuf;
        copied(sb + L.bar_off + 8 * buf, (phases >> buf) & 1);
        phases ^= 1u << buf;
        group_sync(group);                          // everybody is done with the other buffer
        if (tile + 2 < t1 && warp == 0) issue(tile + 2, buf ^ 1);
        float s[4][4] = {};
#pragma unroll
        for (int i = 0; i < kDecSteps; ++i) {
            const int k0 = (warp + 8 * i) * 16;
            if (k0 < Dp) {
                const uint32_t ka = kb + ((lane & 7) + (lane >> 4) * 8) * L.row + (k0 + ((lane >> 3) & 1) * 8) * 2;
                uint32_t b[2][4];
                ldsm4(ka, b[0]);
                ldsm4(ka + 16 * L.row, b[1]);
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    mma_bf16(s[2 * j], qh[i][0], qh[i][1], qh[i][2], qh[i][3], b[j][0], b[j][1]);
                    mma_bf16(s[2 * j + 1], qh[i][0], qh[i][1], qh[i][2], qh[i][3], b[j][2], b[j][3]);
                }
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    mma_bf16(s[2 * j], ql[i][0], ql[i][1], ql[i][2], ql[i][3], b[j][0], b[j][1]);
                    mma_bf16(s[2 * j + 1], ql[i][0], ql[i][1], ql[i][2], ql[i][3], b[j][2], b[j][3]);
                }
            }
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            float* p = part + (warp * 16 + g) * kDecS + 8 * j + 2 * q4;
            *reinterpret_cast<float2*>(p) = make_float2(s[j][0], s[j][1]);
            *reinterpret_cast<float2*>(p + 8 * kDecS) = make_float2(s[j][2], s[j][3]);
        }
        group_sync(group);
        float2 x = make_float2(0.f, 0.f);
#pragma unroll
        for (int w = 0; w < 8; ++w) {
            const float2 y = *reinterpret_cast<const float2*>(part + (w * 16 + srow) * kDecS + skey);
            x.x += y.x;
            x.y += y.y;
        }
        const int key = tile * kDecKeys + skey;
        x.x = key < len ? x.x * a.scale : -INFINITY;
        x.y = key + 1 < len ? x.y * a.scale : -INFINITY;
        float mx = fmaxf(x.x, x.y);
#pragma unroll
        for (int o = 1; o < 16; o <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        mx = fmaxf(mx, m);                          // finite: the first key of a tile is always visible
        const float alpha = expf(m - mx);
        m = mx;
        x.x = expf(x.x - mx);
        x.y = expf(x.y - mx);
        l = l * alpha + (x.x + x.y);
        uint32_t hi, lo;
        split_bf16(x.x, x.y, hi, lo);
        *reinterpret_cast<uint32_t*>(smem + L.p_off + srow * kDecP + skey * 2) = hi;
        *reinterpret_cast<uint32_t*>(smem + L.p_off + (16 + srow) * kDecP + skey * 2) = lo;
        if ((t & 15) == 0) alphas[srow] = alpha;
        group_sync(group);
        const float al0 = alphas[g], al1 = alphas[g + 8];
        if (__any_sync(0xffffffffu, al0 != 1.f || al1 != 1.f)) {
#pragma unroll
            for (int j = 0; j < NT; ++j) { O[j][0] *= al0; O[j][1] *= al0; O[j][2] *= al1; O[j][3] *= al1; }
        }
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
    }
    // the second group hands its result to the first through its key buffers
#pragma unroll
    for (int o = 1; o < 16; o <<= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
    if ((t & 15) == 0) { alphas[srow] = m; alphas[16 + srow] = l; }
    float* other = reinterpret_cast<float*>(smem_all + L.group);
    __syncthreads();   // both groups are done with their keys
    if (group == 1) {
#pragma unroll
        for (int j = 0; j < NT; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) other[(4 * j + i) * 256 + t] = O[j][i];
    }
    __syncthreads();
    if (group == 1) return;
    const float* second = reinterpret_cast<const float*>(smem_all + L.group + L.f_off);
#pragma unroll
    for (int p = 0; p < 2; ++p) {
        const int hr = g + 8 * p, h = h0 + hr;
        if (h >= a.heads) continue;
        const float ma = alphas[hr], mb = second[hr], mm = fmaxf(ma, mb), fa = expf(ma - mm), fb = expf(mb - mm);
        float* out = part_ptr(a, row, h, split);
#pragma unroll
        for (int j = 0; j < NT; ++j) {
            const int col = (warp * NT + j) * 8 + 2 * q4;
            if (col < R8)
                *reinterpret_cast<float2*>(out + col) = make_float2(O[j][2 * p] * fa + other[(4 * j + 2 * p) * 256 + t] * fb,
                                                                    O[j][2 * p + 1] * fa + other[(4 * j + 2 * p + 1) * 256 + t] * fb);
        }
        if (warp == 0 && q4 == 0) {
            out[R8] = mm;
            out[R8 + 1] = alphas[16 + hr] * fa + second[16 + hr] * fb;
        }
    }
}

constexpr int kOutV = 32;   // value columns per block

// Block (head and 32 value columns, RB rows): merges the splits, adds the sink to the denominator, applies W_uv and the gate.
// A warp has four value columns; their first weights are fetched before the kernel waits for its predecessor.
template <typename A, int RB>
__global__ void __launch_bounds__(256) latent_out_kernel(const LatentArgs a, const Rows r, int keys) {
    extern __shared__ float sm[];
    const int R8 = pad8(a.R), dim8 = pad8(a.dim), V8 = pad8(a.V), nq = R8 / 4;
    float* lat = sm;                     // [RB][R8]
    float* wsp = lat + RB * R8;          // [RB][splits] weights of the splits
    float* red = wsp + ((RB * a.splits + 3) & ~3);   // [RB][R8], second half of the splits
    const int vblocks = (V8 + kOutV - 1) / kOutV;
    const int h = blockIdx.x / vblocks, v0 = (blockIdx.x - h * vblocks) * kOutV, row0 = blockIdx.y * RB;
    const int t = threadIdx.x, warp = t >> 5, lane = t & 31;
    const bf16* W = a.Wkv + ((long)a.heads * dim8 + (long)h * V8) * a.ldw;
    pdl_trigger();
    constexpr int kVs = kOutV / 8, kPre = 2;
    uint4 pre[kVs][kPre];
#pragma unroll
    for (int i = 0; i < kVs; ++i)
#pragma unroll
        for (int j = 0; j < kPre; ++j) {
            const int v = v0 + warp + 8 * i, c = lane * 8 + 256 * j;
            pre[i][j] = v < a.V && c < R8 ? __ldg(reinterpret_cast<const uint4*>(W + (long)v * a.ldw + c)) : make_uint4(0, 0, 0, 0);
        }
    pdl_wait();
    if (warp < RB && row0 + warp < r.T) {
        const int row = row0 + warp, ns = r.slot_of(row) < 0 ? 0 : used_splits(min(r.pos_of(row) + 1, a.max_seq), keys, a.splits);
        const float sink = a.sink[h];
        float m = sink;
        for (int s = lane; s < ns; s += 32) m = fmaxf(m, part_ptr(a, row, h, s)[R8]);
        m = warp_max(m);
        float l = 0.f;
        for (int s = lane; s < ns; s += 32) {
            const float* p = part_ptr(a, row, h, s) + R8;
            const float w = expf(p[0] - m);
            wsp[warp * a.splits + s] = w;
            l = fmaf(w, p[1], l);
        }
        l = warp_sum(l) + expf(sink - m);
        __syncwarp();
        for (int s = lane; s < ns; s += 32) wsp[warp * a.splits + s] /= l;
    }
    __syncthreads();
    const int halves = nq <= 128 ? 2 : 1, part = halves == 2 ? t >> 7 : 0;
    for (int i = halves == 2 ? t & 127 : t; i < RB * nq; i += 256 / halves) {
        const int b = i / nq, c = (i - b * nq) * 4, row = row0 + b;
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
        if (row < r.T) {
            const int ns = r.slot_of(row) < 0 ? 0 : used_splits(min(r.pos_of(row) + 1, a.max_seq), keys, a.splits);
            const float* p = part_ptr(a, row, h, 0) + c;
            const long step = R8 + kPartStats;
#pragma unroll 8
            for (int s = part; s < ns; s += halves) {
                const float w = wsp[b * a.splits + s];
                const float4 x = *reinterpret_cast<const float4*>(p + s * step);
                acc.x = fmaf(w, x.x, acc.x);
                acc.y = fmaf(w, x.y, acc.y);
                acc.z = fmaf(w, x.z, acc.z);
                acc.w = fmaf(w, x.w, acc.w);
            }
        }
        *reinterpret_cast<float4*>((part ? red : lat) + b * R8 + c) = acc;
    }
    __syncthreads();
    // sum of the halves, stored as [row][4-column half][8-column block][4]: neighbouring lanes read neighbouring words
    float* lat2 = red + RB * R8;
    for (int i = t; i < RB * R8; i += 256) {
        const int b = i / R8, c = i - b * R8;
        lat2[b * R8 + ((c >> 2) & 1) * (R8 / 2) + (c >> 3) * 4 + (c & 3)] = halves == 2 ? lat[i] + red[i] : lat[i];
    }
    __syncthreads();
    float acc[kVs * RB] = {};
    auto add = [&](const uint4 (&w)[kVs], int c) {
#pragma unroll
        for (int b = 0; b < RB; ++b) {
            const float4 x0 = *reinterpret_cast<const float4*>(lat2 + b * R8 + (c >> 1));
            const float4 x1 = *reinterpret_cast<const float4*>(lat2 + b * R8 + R8 / 2 + (c >> 1));
#pragma unroll
            for (int i = 0; i < kVs; ++i) {
                float s = acc[i * RB + b];
                s = fmaf(x0.x, __uint_as_float(w[i].x << 16), s);
                s = fmaf(x0.y, __uint_as_float(w[i].x & 0xFFFF0000u), s);
                s = fmaf(x0.z, __uint_as_float(w[i].y << 16), s);
                s = fmaf(x0.w, __uint_as_float(w[i].y & 0xFFFF0000u), s);
                s = fmaf(x1.x, __uint_as_float(w[i].z << 16), s);
                s = fmaf(x1.y, __uint_as_float(w[i].z & 0xFFFF0000u), s);
                s = fmaf(x1.z, __uint_as_float(w[i].w << 16), s);
                s = fmaf(x1.w, __uint_as_float(w[i].w & 0xFFFF0000u), s);
                acc[i * RB + b] = s;
            }
        }
    };
#pragma unroll
    for (int j = 0; j < kPre; ++j)
        if (lane * 8 + 256 * j < R8) {
            uint4 w[kVs];
#pragma unroll
            for (int i = 0; i < kVs; ++i) w[i] = pre[i][j];
            add(w, lane * 8 + 256 * j);
        }
    for (int c = lane * 8 + 256 * kPre; c < R8; c += 256) {
        uint4 w[kVs];
#pragma unroll
        for (int i = 0; i < kVs; ++i) {
            const int v = v0 + warp + 8 * i;
            w[i] = v < a.V ? __ldg(reinterpret_cast<const uint4*>(W + (long)v * a.ldw + c)) : make_uint4(0, 0, 0, 0);
        }
        add(w, c);
    }
    const float s = warp_sum_many<kVs * RB>(acc, lane);   // lane -> one (value column, row)
    const int idx = warp_sum_many_index<kVs * RB>(lane), v = v0 + warp + 8 * (idx / RB), row = row0 + idx % RB;
    constexpr int kSpread = 32 / (kVs * RB);              // lanes that hold the same sum
    if (lane % kSpread == 0 && v < V8 && row < r.T)
        static_cast<A*>(a.out)[(long)row * a.ldout + h * V8 + v] =
            from_f<A>(v < a.V ? s * sigmoid_f(a.gate[(long)row * a.ld32 + h]) : 0.f);
}

// ------------------------------------------------------------------------------------------ expanded form
constexpr int kFlashK = 64;   // keys per shared-memory tile
struct FlashSmem {
    int row, vrow, k_off, kbuf, total;
    __host__ __device__ FlashSmem(int D, int VT, int MT) {
        row = D * 2 + 16;
        vrow = VT * 16 + 16;
        k_off = 128 * MT * row;
        kbuf = kFlashK * (row + vrow);
        total = k_off + 2 * kbuf;
    }
};

// Block (128 * MT query rows, head, slice of VT * 8 value columns); a warp has MT tiles of 16 rows, so that every key and
// value fragment it reads from shared memory serves MT products.  MT == 2 takes the 64 keys of a tile in two halves.
template <int VT, int MT>
__global__ void __launch_bounds__(256, 1) latent_flash_kernel(const LatentArgs a, const Rows r) {
    extern __shared__ __align__(16) unsigned char smem[];
    constexpr int kQ = 128 * MT, KT = MT == 1 ? 8 : 4;     // KT: 8-key tiles per softmax step
    const int dim8 = pad8(a.dim), rot8 = pad8(a.rot), D8 = dim8 + rot8, D = pad16(D8), V8 = pad8(a.V), R8 = pad8(a.R);
    const FlashSmem L(D, VT, MT);
    const int t = threadIdx.x, warp = t >> 5, lane = t & 31, g = lane >> 2, q4 = lane & 3;
    // heads fastest, longest rows first
    const int q0 = ((int)gridDim.y - 1 - (int)blockIdx.y) * kQ, h = blockIdx.x, v0 = blockIdx.z * VT * 8;
    const uint32_t sb = smem_u32(smem);
    const bf16* kv = static_cast<const bf16*>(a.kv);
    const long ldkv = (long)a.heads * (dim8 + V8);
    const bf16* kr = static_cast<const bf16*>(a.cache) + (long)r.slot * a.max_seq * a.ldc + R8;
    const int last = min(r.T, q0 + kQ) - 1;                // last real query row of the block
    const int nkeys = r.pos0 + last + 1, tiles = (nkeys + kFlashK - 1) / kFlashK;
    pdl_trigger();
    pdl_wait();
    const int nc = D / 8;
    const RowWalk kwalk(t, 256, nc);
    auto issue = [&](int tile, int buf) {
        const uint32_t kb = sb + L.k_off + buf * L.kbuf, vb = kb + kFlashK * L.row;
        for (RowWalk w = kwalk; w.row < kFlashK; w.next()) {
            const int c = w.col * 8, key = tile * kFlashK + w.row;
            const bool ok = key < nkeys && c < D8;
            const bf16* src = c < dim8 ? kv + (long)key * ldkv + h * dim8 + c : kr + (long)key * a.ldc + (c - dim8);
            cp_async16z(kb + w.row * L.row + c * 2, ok ? src : kv, ok);
        }
        const int vc = (t % VT) * 8;                       // 256 is a multiple of VT: the column stays
        const bool vok = v0 + vc < V8;
        const bf16* vsrc = kv + a.heads * dim8 + h * V8 + v0 + vc;
#pragma unroll
        for (int k = t / VT; k < kFlashK; k += 256 / VT) {
            const int key = tile * kFlashK + k;
            const bool ok = vok && key < nkeys;
            cp_async16z(vb + k * L.vrow + vc * 2, ok ? vsrc + (long)key * ldkv : kv, ok);
        }
        cp_async_commit();
    };
    for (RowWalk w = kwalk; w.row < kQ; w.next()) {
        const bool ok = q0 + w.row < r.T && w.col * 8 < D8;
        const bf16* src = static_cast<const bf16*>(a.q);
        cp_async16z(sb + w.row * L.row + w.col * 16, ok ? src + (long)(q0 + w.row) * a.ldq + h * D8 + w.col * 8 : src, ok);
    }
    issue(0, 0);
    float O[MT][VT][4] = {};
    float m[MT][2], l[MT][2];
#pragma unroll
    for (int i = 0; i < MT; ++i) { m[i][0] = m[i][1] = -INFINITY; l[i][0] = l[i][1] = 0.f; }
    const int wrow = q0 + 16 * MT * warp;                  // first query row of the warp
    const float sl2 = a.scale * 1.4426950408889634f;       // softmax in base 2
    for (int tile = 0; tile < tiles; ++tile) {
        const int buf = tile & 1;
        const uint32_t kb = sb + L.k_off + buf * L.kbuf, vb = kb + kFlashK * L.row;
        cp_async_wait<0>();
        __syncthreads();
        if (tile + 1 < tiles) issue(tile + 1, buf ^ 1);
#pragma unroll 1
        for (int sub = 0; sub < kFlashK; sub += 8 * KT) {
            const int key0 = tile * kFlashK + sub;
            if (key0 > r.pos0 + wrow + 16 * MT - 1) break;  // nothing more of this tile is visible to the warp
            float s[MT][KT][4] = {};
#pragma unroll 2
            for (int k0 = 0; k0 < D; k0 += 16) {
                uint32_t fa[MT][4];
#pragma unroll
                for (int i = 0; i < MT; ++i)
                    ldsm4(sb + (16 * (MT * warp + i) + (lane & 15)) * L.row + (k0 + (lane >> 4) * 8) * 2, fa[i]);
#pragma unroll
                for (int jj = 0; jj < KT / 2; ++jj) {
                    uint32_t fb[4];
                    ldsm4(kb + (sub + 16 * jj + (lane & 7) + (lane >> 4) * 8) * L.row + (k0 + ((lane >> 3) & 1) * 8) * 2, fb);
#pragma unroll
                    for (int i = 0; i < MT; ++i) {
                        mma_bf16(s[i][2 * jj], fa[i][0], fa[i][1], fa[i][2], fa[i][3], fb[0], fb[1]);
                        mma_bf16(s[i][2 * jj + 1], fa[i][0], fa[i][1], fa[i][2], fa[i][3], fb[2], fb[3]);
                    }
                }
            }
            const bool edge = key0 + 8 * KT - 1 > r.pos0 + wrow;
#pragma unroll
            for (int i = 0; i < MT; ++i)
#pragma unroll
                for (int p = 0; p < 2; ++p) {
                    const int pos = r.pos0 + wrow + 16 * i + g + 8 * p;
                    float mx = m[i][p];
#pragma unroll
                    for (int j = 0; j < KT; ++j)
#pragma unroll
                        for (int e = 0; e < 2; ++e) {
                            float& x = s[i][j][2 * p + e];
                            x *= sl2;
                            if (edge && key0 + 8 * j + 2 * q4 + e > pos) x = -INFINITY;
                            mx = fmaxf(mx, x);
                        }
                    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
                    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
                    const float base = mx == -INFINITY ? 0.f : mx, alpha = exp2_fast(m[i][p] - base);
                    m[i][p] = mx;
                    float sum = 0.f;
#pragma unroll
                    for (int j = 0; j < KT; ++j)
#pragma unroll
                        for (int e = 0; e < 2; ++e) {
                            float& x = s[i][j][2 * p + e];
                            x = exp2_fast(x - base);
                            sum += x;
                        }
                    l[i][p] = l[i][p] * alpha + sum;
                    if (__any_sync(0xffffffffu, alpha != 1.f)) {
#pragma unroll
                        for (int j = 0; j < VT; ++j) { O[i][j][2 * p] *= alpha; O[i][j][2 * p + 1] *= alpha; }
                    }
                }
#pragma unroll
            for (int kk = 0; kk < KT / 2; ++kk) {   // 16 keys: the score fragments are the A operand
                uint32_t ph[MT][4], pl[MT][4];
#pragma unroll
                for (int i = 0; i < MT; ++i) {
                    split_bf16(s[i][2 * kk][0], s[i][2 * kk][1], ph[i][0], pl[i][0]);
                    split_bf16(s[i][2 * kk][2], s[i][2 * kk][3], ph[i][1], pl[i][1]);
                    split_bf16(s[i][2 * kk + 1][0], s[i][2 * kk + 1][1], ph[i][2], pl[i][2]);
                    split_bf16(s[i][2 * kk + 1][2], s[i][2 * kk + 1][3], ph[i][3], pl[i][3]);
                }
#pragma unroll
                for (int j = 0; j < VT; j += 2) {
                    uint32_t v[4];
                    ldsm4t(vb + (sub + 16 * kk + (lane & 15)) * L.vrow + (8 * j + (lane >> 4) * 8) * 2, v);
#pragma unroll
                    for (int i = 0; i < MT; ++i) {
                        mma_bf16(O[i][j], ph[i][0], ph[i][1], ph[i][2], ph[i][3], v[0], v[1]);
                        mma_bf16(O[i][j + 1], ph[i][0], ph[i][1], ph[i][2], ph[i][3], v[2], v[3]);
                        mma_bf16(O[i][j], pl[i][0], pl[i][1], pl[i][2], pl[i][3], v[0], v[1]);
                        mma_bf16(O[i][j + 1], pl[i][0], pl[i][1], pl[i][2], pl[i][3], v[2], v[3]);
                    }
                }
            }
        }
    }
    const float sink = a.sink[h] * 1.4426950408889634f;
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int p = 0; p < 2; ++p) {
            const int q = wrow + 16 * i + g + 8 * p;
            float tot = l[i][p];
            tot += __shfl_xor_sync(0xffffffffu, tot, 1);
            tot += __shfl_xor_sync(0xffffffffu, tot, 2);
            if (q >= r.T) continue;
            const float mm = fmaxf(m[i][p], sink), sc = exp2f(m[i][p] - mm);
            const float f = sc / (tot * sc + exp2f(sink - mm)) * sigmoid_f(a.gate[(long)q * a.ld32 + h]);
            bf16* out = static_cast<bf16*>(a.out) + (long)q * a.ldout + h * V8 + v0;
#pragma unroll
            for (int j = 0; j < VT; ++j) {
                const int col = 8 * j + 2 * q4;
                if (v0 + col < V8) *reinterpret_cast<uint32_t*>(out + col) = pack_bf16(O[i][j][2 * p] * f, O[i][j][2 * p + 1] * f);
            }
        }
}

}  // namespace lm
}  // namespace bw
