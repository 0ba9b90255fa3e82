// Launchers of the latent-cache attention.
#include <cuda_runtime.h>

#include <mutex>

#include "../../include/blackwell_b200.h"
#include "host_util.h"
#include "latent_attention.cuh"

namespace bw {
namespace lm {
namespace {

template <typename F>
cudaError_t allow_smem(F kern, std::once_flag (&once)[kMaxDevices]) {
    cudaError_t e = cudaSuccess;
    std::call_once(once[current_device()], [&] { e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxDynSmem); });
    return e;
}

template <typename A, int RB, int COLS>
cudaError_t prep(const LatentArgs& a, const Rows& r, cudaStream_t st) {
    static std::once_flag once[kMaxDevices];
    auto kern = latent_prep_kernel<A, RB, COLS>;
    cudaError_t e = allow_smem(kern, once);
    if (e != cudaSuccess) return e;
    const int cblocks = (pad8(a.R) + COLS - 1) / COLS;
    const size_t smem = (size_t)(RB * (pad8(a.dim) + pad8(a.rot)) + 8 * RB * kPrepThreads) * 4;
    if (smem > kMaxDynSmem) return cudaErrorInvalidValue;
    count_launch(1);
    return launch_pdl(kern, dim3(a.heads * cblocks + (a.dkv ? RB : 0), (r.T + RB - 1) / RB), dim3(kPrepThreads), smem, st, a, r);
}

template <typename A, int RB>
cudaError_t out(const LatentArgs& a, const Rows& r, int keys, cudaStream_t st) {
    static std::once_flag once[kMaxDevices];
    cudaError_t e = allow_smem(latent_out_kernel<A, RB>, once);
    if (e != cudaSuccess) return e;
    const size_t smem = (size_t)(3 * RB * pad8(a.R) + ((RB * a.splits + 3) & ~3)) * 4;
    if (smem > kMaxDynSmem) return cudaErrorInvalidValue;
    count_launch(1);
    return launch_pdl(latent_out_kernel<A, RB>, dim3(a.heads * ((pad8(a.V) + kOutV - 1) / kOutV), (r.T + RB - 1) / RB), dim3(256), smem, st, a, r, keys);
}

template <typename A>
cudaError_t scalar(const LatentArgs& a, const Rows& r, cudaStream_t st) {
    const size_t smem = (size_t)(latent_dp(a.R, a.rot) + kScalarKeys) * 4;
    count_launch(1);
    return launch_pdl(latent_scalar_kernel<A>, dim3(a.splits, a.heads, r.T), dim3(256), smem, st, a, r);
}

template <int NT>
cudaError_t decode(const LatentArgs& a, const Rows& r, cudaStream_t st) {
    static std::once_flag once[kMaxDevices];
    cudaError_t e = allow_smem(latent_decode_kernel<NT>, once);
    if (e != cudaSuccess) return e;
    count_launch(1);
    return launch_pdl(latent_decode_kernel<NT>, dim3(a.splits, (a.heads + 15) / 16, r.T), dim3(kDecThreads), DecodeSmem(a.R, a.rot).total,
                      st, a, r, status_word_ptr());
}

template <int VT, int MT>
cudaError_t flash(const LatentArgs& a, const Rows& r, cudaStream_t st) {
    static std::once_flag once[kMaxDevices];
    auto kern = latent_flash_kernel<VT, MT>;
    cudaError_t e = allow_smem(kern, once);
    if (e != cudaSuccess) return e;
    const int D = pad16(pad8(a.dim) + pad8(a.rot));
    count_launch(1);
    return launch_pdl(kern, dim3(a.heads, (r.T + 128 * MT - 1) / (128 * MT), (pad8(a.V) + VT * 8 - 1) / (VT * 8)), dim3(256),
                      FlashSmem(D, VT, MT).total, st, a, r);
}

// value columns / 8 per block, 0 if no form fits shared memory
int flash_vt(const LatentArgs& a) {
    const int D = pad16(pad8(a.dim) + pad8(a.rot));
    int vt = a.V <= 64 ? 8 : a.V <= 128 ? 16 : 32;
    while (vt > 8 && FlashSmem(D, vt, 1).total > kMaxDynSmem) vt /= 2;
    return FlashSmem(D, vt, 1).total <= kMaxDynSmem ? vt : 0;
}

}  // namespace

bool latent_absorbed_supported(const LatentArgs& a) {
    return a.R >= 1 && a.R <= 2048 && (size_t)(pad8(a.dim) + pad8(a.rot) + 8 * kPrepThreads) * 4 <= (size_t)kMaxDynSmem;
}
bool latent_expanded_supported(const LatentArgs& a) { return flash_vt(a) > 0; }

cudaError_t latent_absorbed(const LatentArgs& a, const Rows& r, int f32, cudaStream_t st) {
    const bool rb4 = r.T >= 8 && !f32 && a.R <= 1024 && (pad8(a.dim) + pad8(a.rot)) <= 1024;
    cudaError_t e = f32 ? prep<float, 1, 64>(a, r, st) : rb4 ? prep<bf16, 4, 256>(a, r, st) : prep<bf16, 1, 64>(a, r, st);
    if (e != cudaSuccess) return e;
    const bool by_scalar = f32 || a.R > 512 || latent_dp(a.R, a.rot) > kDecSteps * 128 || DecodeSmem(a.R, a.rot).total > kMaxDynSmem;
    if (f32) e = scalar<float>(a, r, st);
    else if (by_scalar) e = scalar<bf16>(a, r, st);
    else if (a.R <= 128) e = decode<2>(a, r, st);
    else if (a.R <= 256) e = decode<4>(a, r, st);
    else e = decode<8>(a, r, st);
    if (e != cudaSuccess) return e;
    const int keys = by_scalar ? kScalarKeys : kDecKeys;
    return f32 ? out<float, 1>(a, r, keys, st) : rb4 ? out<bf16, 4>(a, r, keys, st) : out<bf16, 1>(a, r, keys, st);
}

cudaError_t latent_expanded(const LatentArgs& a, const Rows& r, cudaStream_t st) {
    if (r.row_slot) return cudaErrorInvalidValue;
    cudaError_t e = cudaSuccess;
    if (a.dkv) {
        count_launch(1);
        e = launch_pdl(latent_cache_kernel<bf16>, dim3(r.T), dim3(128), 0, st, a, r);
        if (e != cudaSuccess) return e;
    }
    if (a.rot_dims >= 2) {
        count_launch(1);
        e = launch_pdl(latent_rotate_q_kernel, dim3((a.heads * (a.rot_dims / 2) + 127) / 128, r.T), dim3(128), 0, st, a, r);
        if (e != cudaSuccess) return e;
    }
    LinearArgs x{};   // keys and values of the whole context
    x.x = static_cast<const bf16*>(a.cache) + (long)r.slot * a.max_seq * a.ldc;
    x.ldx = a.ldc; x.W = a.Wkv; x.ldw = a.ldw; x.T = r.pos0 + r.T; x.K = a.R;
    x.N = a.heads * (pad8(a.dim) + pad8(a.V)); x.y = a.kv; x.ldy = x.N; x.split = x.N;
    e = linear(x, st);
    if (e != cudaSuccess) return e;
    const int vt = flash_vt(a);
    // 256 query rows per block where that still gives every SM a block
    const bool tall = vt <= 16 && FlashSmem(pad16(pad8(a.dim) + pad8(a.rot)), vt, 2).total <= kMaxDynSmem &&
                      (r.T + 255) / 256 * a.heads >= sm_count(current_device());
    if (tall) return vt == 8 ? flash<8, 2>(a, r, st) : flash<16, 2>(a, r, st);
    return vt == 8 ? flash<8, 1>(a, r, st) : vt == 16 ? flash<16, 1>(a, r, st) : vt == 32 ? flash<32, 1>(a, r, st) : cudaErrorInvalidValue;
}

}  // namespace lm
}  // namespace bw

extern "C" int bw_latent_attention(const bw_latent_args* a, const bw_rows* rows, int expanded, int f32, void* stream) {
    if (!a || !rows || rows->T < 1 || a->heads < 1 || a->dim < 1 || a->rot < 1 || a->V < 1 || a->R < 1 || a->rot_dims < 0 ||
        a->rot_dims > a->rot || a->rot_dims % 2 != 0 || !a->cs || !a->cache || !a->q || !a->gate || !a->Wkv || !a->sink || !a->out ||
        (a->dkv && !a->dkv_norm) || a->max_seq < 1 || a->ldc < bw::lm::latent_row(a->R, a->rot) || a->ldc % 8 != 0 || a->ldq % 8 != 0 ||
        a->ldw < bw::lm::pad8(a->R) || a->ldw % 8 != 0 || a->ldout % 8 != 0 || (rows->row_slot && !rows->row_pos) ||
        (!rows->row_slot && rows->pos0 + rows->T > a->max_seq))
        return cudaErrorInvalidValue;
    bw::lm::LatentArgs l{};
    l.heads = a->heads; l.dim = a->dim; l.rot = a->rot; l.V = a->V; l.R = a->R; l.rot_dims = a->rot_dims; l.scale = a->scale; l.eps = a->eps;
    l.cs = static_cast<const float2*>(a->cs); l.max_seq = a->max_seq; l.cache = a->cache; l.ldc = a->ldc; l.q = a->q; l.ldq = a->ldq;
    l.dkv = a->dkv; l.gate = a->gate; l.ld32 = a->ld32; l.dkv_norm = a->dkv_norm; l.Wkv = reinterpret_cast<const bw::lm::bf16*>(a->Wkv);
    l.ldw = a->ldw; l.sink = a->sink; l.out = a->out; l.ldout = a->ldout; l.qabs = a->qabs; l.part = a->part; l.splits = a->splits; l.kv = a->kv;
    const bw::lm::Rows w{rows->T, rows->row_slot, rows->row_pos, rows->slot, rows->pos0};
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (expanded)
        return f32 || !a->kv || !bw::lm::latent_expanded_supported(l) ? cudaErrorInvalidValue : bw::lm::latent_expanded(l, w, st);
    if (!a->qabs || !a->part || a->splits < 1 || !bw::lm::latent_absorbed_supported(l)) return cudaErrorInvalidValue;
    return bw::lm::latent_absorbed(l, w, f32, st);
}
