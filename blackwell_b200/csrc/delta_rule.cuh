// Gated delta rule for prompts (bf16), 64 tokens at a time.  With the decays g, Gamma_i = g_1 ... g_i inside the chunk, S_0 the
// state before it and unit vectors k, q, the writes u_i of a chunk solve a unit lower triangular system:
//   (I + A) U = diag(beta) (V - diag(Gamma) K S_0),   A_ij = beta_i (Gamma_i / Gamma_j) (k_i k_j) for j < i
//   O = diag(Gamma) Q S_0 + P U,   P_ij = (Gamma_i / Gamma_j) (q_i k_j) for j <= i
//   S = Gamma_64 S_0 + sum_j (Gamma_64 / Gamma_j) k_j u_j^T
//   delta_prepare_kernel   what does not depend on the state, all chunks at once: the norms of k and q, the cumulative
//                          decays, T = (I + A)^-1 and P.
//   delta_chunk_kernel     the chunks of a head one after the other, a tile of state columns per CTA, state in registers.
// k, q and v are bf16 values and enter the products (mma.sync) as they are: the unit norms are applied to the fp32 results.
// T, P, the right-hand side, U and the state enter as a bf16 high part plus a bf16 remainder.
#pragma once
#include "recurrence.cuh"

namespace bw {
namespace lm {

// per chunk and head: T high, T remainder, P high, P remainder [64][64], then cumulative log2 decay, beta, 1 / |k|, q_scale / |q|
constexpr int kDeltaMat = kChunk * kChunk * 2;
constexpr int kDeltaUnit = 4 * kDeltaMat + 4 * kChunk * 4;
constexpr int kInvRow = kChunk + 4;   // floats of a row of A^T in shared memory

// q and k, whose place T and a factor take over; A^T; the four vectors
inline __host__ __device__ int delta_prepare_front(int N) {
    const int qk = 2 * kChunk * (pad16(N) * 2 + 16), inv = kChunk * kInvRow * 4 + 32 * 36 * 4;
    return qk > inv ? qk : inv;
}
inline __host__ __device__ int delta_prepare_smem(int N) { return delta_prepare_front(N) + kChunk * kInvRow * 4 + 4 * kChunk * 4; }

// Block (head, chunk).
__global__ void __launch_bounds__(256) delta_prepare_kernel(const RecurrenceArgs a, const Rows r) {
    extern __shared__ __align__(16) unsigned char smem[];
    const int NP = pad16(a.N), N8 = pad8(a.N), qrow = NP * 2 + 16;
    const int t = threadIdx.x, warp = t >> 5, lane = t & 31, g = lane >> 2, q4 = lane & 3;
    const int h = blockIdx.x, ch = blockIdx.y, grp = h / (a.heads / a.groups);
    float* At = reinterpret_cast<float*>(smem + delta_prepare_front(a.N));   // [column of A][row of A]
    float *cum = At + kChunk * kInvRow, *beta = cum + kChunk, *rk = beta + kChunk, *rq = rk + kChunk;
    unsigned char* unit = static_cast<unsigned char*>(a.chunk_scratch) + ((long)ch * a.heads + h) * kDeltaUnit;
    const uint32_t qb = smem_u32(smem), kb = qb + kChunk * qrow;
    const bf16* qg = static_cast<const bf16*>(a.q) + grp * N8;
    const bf16* kg = static_cast<const bf16*>(a.k) + grp * N8;
    pdl_wait();
    for (RowWalk w(t, 256, NP / 8); w.row < kChunk; w.next()) {
        const int col = w.col * 8, tok = ch * kChunk + w.row;
        const bool ok = tok < r.T && col < N8;
        cp_async16z(qb + w.row * qrow + col * 2, ok ? qg + (long)tok * a.ldq + col : qg, ok);
        cp_async16z(kb + w.row * qrow + col * 2, ok ? kg + (long)tok * a.ldk + col : kg, ok);
    }
    cp_async_commit();
    if (warp == 0) {
        float l[2], b[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int tok = ch * kChunk + 2 * lane + i;
            const bool ok = tok < r.T;   // rows past the end: no decay, nothing written
            l[i] = ok ? a.log_decay[(long)tok * a.heads + h] * kLog2e : 0.f;
            b[i] = ok ? a.weight[(long)tok * a.heads + h] : 0.f;
        }
        float s = l[0] + l[1];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, s, o);
            if (lane >= o) s += up;
        }
        *reinterpret_cast<float2*>(cum + 2 * lane) = make_float2(s - l[1], s);
        *reinterpret_cast<float2*>(beta + 2 * lane) = make_float2(b[0], b[1]);
    }
    cp_async_wait<0>();
    __syncthreads();
    for (int i = warp; i < kChunk; i += 8) {
        float sq = 0.f, sk = 0.f;
        for (int c = lane; c < NP / 2; c += 32) {
            const uint32_t x = *reinterpret_cast<const uint32_t*>(smem + i * qrow + c * 4);
            const uint32_t y = *reinterpret_cast<const uint32_t*>(smem + (kChunk + i) * qrow + c * 4);
            const float x0 = __uint_as_float(x << 16), x1 = __uint_as_float(x & 0xFFFF0000u);
            const float y0 = __uint_as_float(y << 16), y1 = __uint_as_float(y & 0xFFFF0000u);
            sq = fmaf(x0, x0, fmaf(x1, x1, sq));
            sk = fmaf(y0, y0, fmaf(y1, y1, sk));
        }
        sq = warp_sum(sq);
        sk = warp_sum(sk);
        if (lane == 0) {
            rk[i] = 1.0f / sqrtf(sk + a.unit_eps);
            rq[i] = a.q_scale / sqrtf(sq + a.unit_eps);
        }
    }
    __syncthreads();

    // q k^T (warps 0-3) and k k^T (warps 4-7), 16 rows each
    const bool isk = warp >= 4;
    const int r0 = 16 * (warp & 3);
    float c[8][4] = {};
    for (int k0 = 0; k0 < NP; k0 += 16) {
        uint32_t fa[4];
        ldsm4((isk ? kb : qb) + (r0 + (lane & 15)) * qrow + (k0 + (lane >> 4) * 8) * 2, fa);
#pragma unroll
        for (int jj = 0; jj < 4; ++jj)
            if (16 * jj <= r0) {
                uint32_t fb[4];
                ldsm4(kb + (16 * jj + (lane & 7) + (lane >> 4) * 8) * qrow + (k0 + ((lane >> 3) & 1) * 8) * 2, fb);
                mma_bf16(c[2 * jj], fa[0], fa[1], fa[2], fa[3], fb[0], fb[1]);
                mma_bf16(c[2 * jj + 1], fa[0], fa[1], fa[2], fa[3], fb[2], fb[3]);
            }
    }
#pragma unroll
    for (int p = 0; p < 2; ++p) {
        const int row = r0 + g + 8 * p;
        const float cr = cum[row], f = isk ? beta[row] * rk[row] : rq[row];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int col = 8 * j + 2 * q4;
            float v[2];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const bool in = isk ? col + e < row : col + e <= row;
                v[e] = in ? c[j][2 * p + e] * exp2_fast(cr - cum[col + e]) * f * rk[col + e] : 0.f;
            }
            if (isk) {
                At[col * kInvRow + row] = v[0];
                At[(col + 1) * kInvRow + row] = v[1];
            } else {
                uint32_t hi, lo;
                split_bf16(v[0], v[1], hi, lo);
                uint32_t* o = reinterpret_cast<uint32_t*>(unit + 2 * kDeltaMat) + (row * kChunk + col) / 2;
                o[0] = hi;
                o[kDeltaMat / 4] = lo;
            }
        }
    }
    for (int i = t; i < 4 * kChunk; i += 256) reinterpret_cast<float*>(unit + 4 * kDeltaMat)[i] = cum[i];
    __syncthreads();
    // T = (I + A)^-1: the 16 x 16 blocks on the diagonal by forward substitution, a thread per column, then twice the block
    // below two inverted ones, T_21 = -T_22 A_21 T_11
    float *T = reinterpret_cast<float*>(smem), *M = T + kChunk * kInvRow;
    for (int i = t; i < kChunk * kInvRow / 4; i += 256) reinterpret_cast<float4*>(T)[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    __syncthreads();
    if (t < kChunk) {
        const int b0 = t & ~15, j = t & 15;
        float x[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) x[i] = i == j ? 1.f : 0.f;
#pragma unroll
        for (int l = 0; l < 16; ++l)
#pragma unroll
            for (int i = (l + 1) / 4 * 4; i < 16; i += 4) {   // A is zero on and above the diagonal
                const float4 v = *reinterpret_cast<const float4*>(At + (b0 + l) * kInvRow + b0 + i);
                x[i] = fmaf(-v.x, x[l], x[i]);
                x[i + 1] = fmaf(-v.y, x[l], x[i + 1]);
                x[i + 2] = fmaf(-v.z, x[l], x[i + 2]);
                x[i + 3] = fmaf(-v.w, x[l], x[i + 3]);
            }
#pragma unroll
        for (int i = 0; i < 16; ++i) T[(b0 + i) * kInvRow + t] = x[i];
    }
    __syncthreads();
    {
        const int b0 = t >> 7 << 5, i = (t >> 3) & 15, j = (t & 7) * 2;
        float* Mp = M + (t >> 7) * 16 * 20;
        float2 s = make_float2(0.f, 0.f);
#pragma unroll
        for (int l = 0; l < 16; ++l) {
            const float x = At[(b0 + l) * kInvRow + b0 + 16 + i];
            const float2 y = *reinterpret_cast<const float2*>(T + (b0 + l) * kInvRow + b0 + j);
            s.x = fmaf(x, y.x, s.x);
            s.y = fmaf(x, y.y, s.y);
        }
        *reinterpret_cast<float2*>(Mp + i * 20 + j) = s;
        __syncthreads();
        s = make_float2(0.f, 0.f);
#pragma unroll
        for (int l = 0; l < 16; ++l) {
            const float x = -T[(b0 + 16 + i) * kInvRow + b0 + 16 + l];
            const float2 y = *reinterpret_cast<const float2*>(Mp + l * 20 + j);
            s.x = fmaf(x, y.x, s.x);
            s.y = fmaf(x, y.y, s.y);
        }
        *reinterpret_cast<float2*>(T + (b0 + 16 + i) * kInvRow + b0 + j) = s;
    }
    __syncthreads();
    {
        const int i = t >> 3, j = (t & 7) * 4;
        auto product = [&](auto left, const float* right, int ld) {
            float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
            for (int l = 0; l < 32; ++l) {
                const float x = left(l);
                const float4 y = *reinterpret_cast<const float4*>(right + l * ld + j);
                s.x = fmaf(x, y.x, s.x);
                s.y = fmaf(x, y.y, s.y);
                s.z = fmaf(x, y.z, s.z);
                s.w = fmaf(x, y.w, s.w);
            }
            return s;
        };
        const float4 mt = product([&](int l) { return At[l * kInvRow + 32 + i]; }, T, kInvRow);
        *reinterpret_cast<float4*>(M + i * 36 + j) = mt;
        __syncthreads();
        *reinterpret_cast<float4*>(T + (32 + i) * kInvRow + j) = product([&](int l) { return -T[(32 + i) * kInvRow + 32 + l]; }, M, 36);
    }
    __syncthreads();
    for (int i = t; i < kChunk * kChunk / 2; i += 256) {
        const float2 x = *reinterpret_cast<const float2*>(T + (i >> 5) * kInvRow + (i & 31) * 2);
        uint32_t hi, lo;
        split_bf16(x.x, x.y, hi, lo);
        reinterpret_cast<uint32_t*>(unit)[i] = hi;
        reinterpret_cast<uint32_t*>(unit + kDeltaMat)[i] = lo;
    }
}

struct DeltaSmem {
    int qrow, vrow, k_off, v_off, m_off, c_off, buf, s_off, r_off, u_off, total;
    __host__ __device__ DeltaSmem(int N, int VT, int nbuf) {
        const int NP = pad16(N);
        qrow = NP * 2 + 16;
        vrow = VT * 2 + 16;
        k_off = kChunk * qrow;
        v_off = 2 * kChunk * qrow;
        m_off = v_off + kChunk * vrow;             // T high, T remainder, P high, P remainder
        c_off = m_off + 4 * kChunk * kPRow;
        buf = c_off + 4 * kChunk * 4;              // one buffer
        s_off = nbuf * buf;                        // state, high and remainder
        r_off = s_off + 2 * NP * vrow;             // right-hand side, high and remainder
        u_off = r_off + 2 * kChunk * vrow;         // U, high and remainder; U weighted by what is left of it at the end
        total = u_off + 4 * kChunk * vrow;
    }
};

// NTW: 16-row state tiles per warp; VT: state columns per CTA (64 or 32).
template <int NTW, int VT>
__global__ void __launch_bounds__(256) delta_chunk_kernel(const RecurrenceArgs a, const Rows r, int nbuf) {
    extern __shared__ __align__(16) unsigned char smem[];
    constexpr int NT = VT / 8;
    const DeltaSmem L(a.N, VT, nbuf);
    const int NP = pad16(a.N), N8 = pad8(a.N), V8 = pad8(a.V);
    const int t = threadIdx.x, warp = t >> 5, lane = t & 31, g = lane >> 2, q4 = lane & 3;
    const int h = blockIdx.y, v0 = blockIdx.x * VT, grp = h / (a.heads / a.groups);
    const uint32_t sb = smem_u32(smem);
    const int nchunks = (r.T + kChunk - 1) / kChunk;
    const bf16* qg = static_cast<const bf16*>(a.q) + grp * N8;
    const bf16* kg = static_cast<const bf16*>(a.k) + grp * N8;
    const bf16* vg = static_cast<const bf16*>(a.v) + h * V8 + v0;
    const unsigned char* units = static_cast<const unsigned char*>(a.chunk_scratch) + (long)h * kDeltaUnit;
    pdl_wait();

    const RowWalk walk(t, 256, NP / 8);
    auto issue = [&](int ch, int buf) {
        const uint32_t base = sb + buf * L.buf;
        for (RowWalk w = walk; w.row < kChunk; w.next()) {
            const int col = w.col * 8, tok = ch * kChunk + w.row;
            const bool ok = tok < r.T && col < N8;
            cp_async16z(base + w.row * L.qrow + col * 2, ok ? qg + (long)tok * a.ldq + col : qg, ok);
            cp_async16z(base + L.k_off + w.row * L.qrow + col * 2, ok ? kg + (long)tok * a.ldk + col : kg, ok);
        }
#pragma unroll
        for (int i = t; i < kChunk * (VT / 8); i += 256) {
            const int row = i / (VT / 8), col = (i % (VT / 8)) * 8, tok = ch * kChunk + row;
            const bool ok = tok < r.T && v0 + col < V8;
            cp_async16z(base + L.v_off + row * L.vrow + col * 2, ok ? vg + (long)tok * a.ldv + col : vg, ok);
        }
        const unsigned char* unit = units + (long)ch * a.heads * kDeltaUnit;
#pragma unroll
        for (int i = t; i < 4 * kChunk * 8; i += 256) cp_async16z(base + L.m_off + (i >> 3) * kPRow + (i & 7) * 16, unit + i * 16, true);
        if (t < kChunk) cp_async16z(base + L.c_off + t * 16, unit + 4 * kDeltaMat + t * 16, true);
        cp_async_commit();
    };

    // state fragments: rows 16 * (i * 8 + warp) .., columns 8 * j ..
    float S[NTW][NT][4];
    float* Sg = a.S + (((long)r.slot * a.heads + h) * a.N) * V8 + v0;
    auto state_to_smem = [&] {
#pragma unroll
        for (int i = 0; i < NTW; ++i) {
            const int n0 = 16 * (i * 8 + warp);
            if (n0 >= NP) continue;
#pragma unroll
            for (int j = 0; j < NT; ++j)
#pragma unroll
                for (int p = 0; p < 2; ++p) {
                    uint32_t hi, lo;
                    split_bf16(S[i][j][2 * p], S[i][j][2 * p + 1], hi, lo);
                    const int off = L.s_off + (n0 + g + 8 * p) * L.vrow + (8 * j + 2 * q4) * 2;
                    *reinterpret_cast<uint32_t*>(smem + off) = hi;
                    *reinterpret_cast<uint32_t*>(smem + off + NP * L.vrow) = lo;
                }
        }
    };
    issue(0, 0);
#pragma unroll
    for (int i = 0; i < NTW; ++i)
#pragma unroll
        for (int j = 0; j < NT; ++j)
#pragma unroll
            for (int p = 0; p < 2; ++p) {
                const int n = 16 * (i * 8 + warp) + g + 8 * p, v = 8 * j + 2 * q4;
                float2 s = make_float2(0.f, 0.f);
                if (r.pos0 > 0 && n < a.N && v0 + v < V8) s = *reinterpret_cast<const float2*>(Sg + (long)n * V8 + v);
                S[i][j][2 * p] = s.x;
                S[i][j][2 * p + 1] = s.y;
            }
    state_to_smem();

    const bool isk = warp >= 4;
    const int r0 = 16 * (warp & 3), o0 = (VT / 2) * (warp >> 2);
    const int lrow = lane & 15, lcol = (lane >> 4) * 8;
    for (int ch = 0; ch < nchunks; ++ch) {
        const int buf = nbuf == 2 ? ch & 1 : 0, off = buf * L.buf;
        const uint32_t qb = sb + off, kb = qb + L.k_off, mb = qb + L.m_off;
        cp_async_wait<0>();
        __syncthreads();   // operands and state copy are in shared memory
        if (nbuf == 2 && ch + 1 < nchunks) issue(ch + 1, buf ^ 1);
        const float *cum = reinterpret_cast<const float*>(smem + off + L.c_off), *beta = cum + kChunk, *rk = beta + kChunk, *rq = rk + kChunk;
        const float total = cum[kChunk - 1];

        // q S_0 (warps 0-3), k S_0 (warps 4-7)
        float acc[NT][4] = {};
#pragma unroll 2
        for (int k0 = 0; k0 < NP; k0 += 16) {
            uint32_t fa[4];
            ldsm4((isk ? kb : qb) + (r0 + lrow) * L.qrow + (k0 + lcol) * 2, fa);
#pragma unroll
            for (int jj = 0; jj < VT / 16; ++jj)
#pragma unroll
                for (int part = 0; part < 2; ++part) {
                    uint32_t fs[4];
                    ldsm4t(sb + L.s_off + (part * NP + k0 + lrow) * L.vrow + (16 * jj + lcol) * 2, fs);
                    mma_bf16(acc[2 * jj], fa[0], fa[1], fa[2], fa[3], fs[0], fs[1]);
                    mma_bf16(acc[2 * jj + 1], fa[0], fa[1], fa[2], fa[3], fs[2], fs[3]);
                }
        }
#pragma unroll
        for (int p = 0; p < 2; ++p) {
            const int row = r0 + g + 8 * p;
            const float f = exp2_fast(cum[row]) * (isk ? rk[row] : rq[row]), b = beta[row];
#pragma unroll
            for (int j = 0; j < NT; ++j) {
                if (isk) {
                    const int col = (8 * j + 2 * q4) * 2;
                    const uint32_t vv = *reinterpret_cast<const uint32_t*>(smem + off + L.v_off + row * L.vrow + col);
                    uint32_t hi, lo;
                    split_bf16(b * (__uint_as_float(vv << 16) - f * acc[j][2 * p]), b * (__uint_as_float(vv & 0xFFFF0000u) - f * acc[j][2 * p + 1]), hi, lo);
                    *reinterpret_cast<uint32_t*>(smem + L.r_off + row * L.vrow + col) = hi;
                    *reinterpret_cast<uint32_t*>(smem + L.r_off + (kChunk + row) * L.vrow + col) = lo;
                } else {
                    acc[j][2 * p] *= f;
                    acc[j][2 * p + 1] *= f;
                }
            }
        }
        __syncthreads();   // right-hand side written, old state copy read

        // U = T R: 16 rows, half of the columns per warp
        float u[NT / 2][4] = {};
        for (int k0 = 0; k0 <= r0; k0 += 16) {
            uint32_t th[4], tl[4];
            ldsm4(mb + (r0 + lrow) * kPRow + (k0 + lcol) * 2, th);
            ldsm4(mb + (kChunk + r0 + lrow) * kPRow + (k0 + lcol) * 2, tl);
#pragma unroll
            for (int jj = 0; jj < VT / 32; ++jj) {
                uint32_t rh[4], rl[4];
                const uint32_t ra = sb + L.r_off + (k0 + lrow) * L.vrow + (o0 + 16 * jj + lcol) * 2;
                ldsm4t(ra, rh);
                ldsm4t(ra + kChunk * L.vrow, rl);
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    mma_bf16(u[2 * jj + e], th[0], th[1], th[2], th[3], rh[2 * e], rh[2 * e + 1]);
                    mma_bf16(u[2 * jj + e], th[0], th[1], th[2], th[3], rl[2 * e], rl[2 * e + 1]);
                    mma_bf16(u[2 * jj + e], tl[0], tl[1], tl[2], tl[3], rh[2 * e], rh[2 * e + 1]);
                }
            }
        }
#pragma unroll
        for (int p = 0; p < 2; ++p) {
            const int row = r0 + g + 8 * p;
            const float left = exp2_fast(total - cum[row]) * rk[row];
#pragma unroll
            for (int j = 0; j < NT / 2; ++j) {
                unsigned char* d = smem + L.u_off + row * L.vrow + (o0 + 8 * j + 2 * q4) * 2;
                uint32_t hi, lo;
                split_bf16(u[j][2 * p], u[j][2 * p + 1], hi, lo);
                *reinterpret_cast<uint32_t*>(d) = hi;
                *reinterpret_cast<uint32_t*>(d + kChunk * L.vrow) = lo;
                split_bf16(u[j][2 * p] * left, u[j][2 * p + 1] * left, hi, lo);
                *reinterpret_cast<uint32_t*>(d + 2 * kChunk * L.vrow) = hi;
                *reinterpret_cast<uint32_t*>(d + 3 * kChunk * L.vrow) = lo;
            }
        }
        __syncthreads();   // U written

        // out += P U (warps 0-3)
        if (!isk) {
            for (int k0 = 0; k0 <= r0; k0 += 16) {
                uint32_t ph[4], pl[4];
                ldsm4(mb + (2 * kChunk + r0 + lrow) * kPRow + (k0 + lcol) * 2, ph);
                ldsm4(mb + (3 * kChunk + r0 + lrow) * kPRow + (k0 + lcol) * 2, pl);
#pragma unroll
                for (int jj = 0; jj < VT / 16; ++jj) {
                    uint32_t uh[4], ul[4];
                    const uint32_t ua = sb + L.u_off + (k0 + lrow) * L.vrow + (16 * jj + lcol) * 2;
                    ldsm4t(ua, uh);
                    ldsm4t(ua + kChunk * L.vrow, ul);
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        mma_bf16(acc[2 * jj + e], ph[0], ph[1], ph[2], ph[3], uh[2 * e], uh[2 * e + 1]);
                        mma_bf16(acc[2 * jj + e], ph[0], ph[1], ph[2], ph[3], ul[2 * e], ul[2 * e + 1]);
                        mma_bf16(acc[2 * jj + e], pl[0], pl[1], pl[2], pl[3], uh[2 * e], uh[2 * e + 1]);
                    }
                }
            }
#pragma unroll
            for (int j = 0; j < NT; ++j)
#pragma unroll
                for (int p = 0; p < 2; ++p) {
                    const int col = 8 * j + 2 * q4, tok = ch * kChunk + r0 + g + 8 * p;
                    if (tok < r.T && v0 + col < V8)
                        *reinterpret_cast<float2*>(a.o + (long)tok * a.ldo + h * V8 + v0 + col) = make_float2(acc[j][2 * p], acc[j][2 * p + 1]);
                }
        }
        // state: S = exp(total) S + k^T (weighted U)
        const float et = exp2_fast(total);
#pragma unroll
        for (int i = 0; i < NTW; ++i) {
            const int n0 = 16 * (i * 8 + warp);
            if (n0 >= NP) continue;
#pragma unroll
            for (int j = 0; j < NT; ++j)
#pragma unroll
                for (int p = 0; p < 4; ++p) S[i][j][p] *= et;
#pragma unroll
            for (int k0 = 0; k0 < kChunk; k0 += 16) {
                uint32_t fk[4];   // k^T: row n, column token
                ldsm4t(kb + (k0 + (lane & 7) + lcol) * L.qrow + (n0 + ((lane >> 3) & 1) * 8) * 2, fk);
#pragma unroll
                for (int jj = 0; jj < VT / 16; ++jj)
#pragma unroll
                    for (int part = 2; part < 4; ++part) {
                        uint32_t fu[4];
                        ldsm4t(sb + L.u_off + (part * kChunk + k0 + lrow) * L.vrow + (16 * jj + lcol) * 2, fu);
                        mma_bf16(S[i][2 * jj], fk[0], fk[1], fk[2], fk[3], fu[0], fu[1]);
                        mma_bf16(S[i][2 * jj + 1], fk[0], fk[1], fk[2], fk[3], fu[2], fu[3]);
                    }
            }
        }
        state_to_smem();
        if (nbuf == 1) {
            __syncthreads();
            if (ch + 1 < nchunks) issue(ch + 1, 0);
        }
    }
#pragma unroll
    for (int i = 0; i < NTW; ++i)
#pragma unroll
        for (int j = 0; j < NT; ++j)
#pragma unroll
            for (int p = 0; p < 2; ++p) {
                const int n = 16 * (i * 8 + warp) + g + 8 * p, v = 8 * j + 2 * q4;
                if (n < a.N && v0 + v < V8)
                    *reinterpret_cast<float2*>(Sg + (long)n * V8 + v) = make_float2(S[i][j][2 * p], S[i][j][2 * p + 1]);
            }
}

}  // namespace lm
}  // namespace bw
