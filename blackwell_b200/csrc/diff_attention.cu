// Launchers of the differential attention.
#include <cuda_runtime.h>

#include <algorithm>
#include <mutex>

#include "../../include/blackwell_b200.h"
#include "diff_attention.cuh"
#include "host_util.h"
#include "tensor_map.h"

namespace bw {
namespace lm {
namespace {

template <typename F>
cudaError_t allow_smem(F kern, std::once_flag (&once)[kMaxDevices]) {
    cudaError_t e = cudaSuccess;
    std::call_once(once[current_device()], [&] { e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxDynSmem); });
    return e;
}

int decode_blocks(const DiffAttnArgs& a, int rows) { return a.kv_heads * ((a.heads / a.kv_heads + 7) / 8) * rows; }

template <typename A, int VW>
cudaError_t prep(const DiffAttnArgs& a, const Rows& r, cudaStream_t st) {
    const int half = a.rot_dims / 2;
    int items = a.heads * 2 * (half / VW);
    if (a.k) items += a.kv_heads * (2 * (half / VW) + 2 * ((pad8(a.dim) - a.rot_dims) / VW) + pad8(a.V) / VW);
    if (items == 0) return cudaSuccess;
    count_launch(1);
    return launch_pdl(diff_prep_kernel<A, VW>, dim3((items + 255) / 256, r.T), dim3(256), 0, st, a, r);
}

template <typename A>
cudaError_t scalar(const DiffAttnArgs& a, const Rows& r, cudaStream_t st) {
    const size_t smem = (size_t)(2 * pad8(a.dim) + 2 * kDiffKeys + 32) * 4;
    count_launch(1);
    return launch_pdl(diff_scalar_kernel<A>, dim3(a.heads, r.T), dim3(256), smem, st, a, r);
}

template <int KS, int VT, int WARPS>
cudaError_t decode_inst(const DiffAttnArgs& a, const Rows& r, cudaStream_t st) {
    static std::once_flag once[kMaxDevices];
    auto kern = diff_decode_kernel<KS, VT, WARPS>;
    cudaError_t e = allow_smem(kern, once);
    if (e != cudaSuccess) return e;
    int stages = 4;
    while (stages > 2 && DiffDecodeSmem(a.dim, a.V, VT, WARPS, stages).total > (WARPS == 4 ? 113 * 1024 : kMaxDynSmem)) --stages;   // two blocks of four warps per SM
    const int smem = DiffDecodeSmem(a.dim, a.V, VT, WARPS, stages).total, group = a.heads / a.kv_heads;
    const int ldc = a.kv_heads * diff_row(a.dim, a.V);
    CUtensorMap map;
    if (!make_map(&map, a.cache, ldc, (long)a.slots * a.cap, ldc, kDiffTile)) return cudaErrorInvalidValue;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(a.splits, a.kv_heads * ((group + 7) / 8), r.T);
    cfg.blockDim = dim3(WARPS * 32);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = pdl_enabled() ? 1 : 0;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = a.splits;
    attr[1].val.clusterDim.y = 1;
    attr[1].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 2;
    count_launch(1);
    return cudaLaunchKernelEx(&cfg, kern, map, a, r, stages, status_word_ptr());
}
template <int KS, int VT>
cudaError_t decode(const DiffAttnArgs& a, const Rows& r, cudaStream_t st) {
    // eight warps per block while the blocks do not even fill the SMs once
    const bool few = decode_blocks(a, r.T) * a.splits <= sm_count(current_device()) && DiffDecodeSmem(a.dim, a.V, VT, 8, 2).total <= kMaxDynSmem;
    return few ? decode_inst<KS, VT, 8>(a, r, st) : decode_inst<KS, VT, 4>(a, r, st);
}

template <int VT, int MT, int KK>
cudaError_t flash(const DiffAttnArgs& a, const Rows& r, cudaStream_t st) {
    static std::once_flag once[kMaxDevices];
    auto kern = diff_flash_kernel<VT, MT, KK>;
    cudaError_t e = allow_smem(kern, once);
    if (e != cudaSuccess) return e;
    count_launch(1);
    return launch_pdl(kern, dim3(a.heads, (r.T + 64 * MT - 1) / (64 * MT)), dim3(256), DiffFlashSmem(a.dim, VT, MT, KK).total, st, a, r);
}

// Sizes of the tensor-core kernels: the smallest instance that holds them, 0 if none does.
int decode_size(const DiffAttnArgs& a) {
    const int size = std::max(pad16(a.dim), pad8(a.V));
    const int s = size <= 64 ? 64 : size <= 128 ? 128 : size <= 256 ? 256 : 0;
    return s && DiffDecodeSmem(a.dim, a.V, s / 8, 4, 2).total <= kMaxDynSmem ? s : 0;
}
template <int VT, int MT, int KK>
bool flash_fits(const DiffAttnArgs& a) { return pad8(a.V) <= VT * 8 && DiffFlashSmem(a.dim, VT, MT, KK).total <= kMaxDynSmem; }

}  // namespace

bool diff_attention_supported(const DiffAttnArgs& a) {
    return a.heads >= 1 && a.kv_heads >= 1 && a.heads % a.kv_heads == 0 && a.dim >= 1 && a.dim <= 4096 && a.V >= 1 && a.V <= 8 * 256 &&
           a.window >= 0 && a.rot_dims >= 0 && a.rot_dims <= a.dim && a.rot_dims % 2 == 0;
}

int diff_attention_splits(const DiffAttnArgs& a, int rows, int f32) {
    if (f32 || !decode_size(a)) return 1;
    // two blocks per SM, at least two tiles per warp of four at full length
    const int blocks = decode_blocks(a, rows), sms = sm_count(current_device());
    const int len = a.window > 0 ? std::min(a.window, a.max_seq) : a.max_seq, tiles = (len + kDiffTile - 1) / kDiffTile;
    int s = 1;
    while (s < 8 && 2 * s * blocks <= 2 * sms && tiles >= 16 * s) s *= 2;
    return s;
}

cudaError_t diff_attention(const DiffAttnArgs& a, const Rows& r, int f32, cudaStream_t st) {
    if (r.T < 1 || !diff_attention_supported(a)) return cudaErrorInvalidValue;
    if (f32) {
        const cudaError_t e = prep<float, 1>(a, r, st);
        return e != cudaSuccess ? e : scalar<float>(a, r, st);
    }
    if (r.row_slot && (a.splits == 1 || a.splits == 2 || a.splits == 4 || a.splits == 8)) {
        const int size = decode_size(a);
        if (size == 64) return decode<4, 8>(a, r, st);
        if (size == 128) return decode<8, 16>(a, r, st);
        if (size == 256) return decode<16, 32>(a, r, st);
    }
    const cudaError_t e = a.rot_dims % 16 == 0 ? prep<bf16, 8>(a, r, st) : prep<bf16, 1>(a, r, st);
    if (e != cudaSuccess || r.row_slot) return e != cudaSuccess ? e : scalar<bf16>(a, r, st);
    // 128 query rows per block where that still gives every SM a block
    const bool tall = (r.T + 127) / 128 * a.heads >= sm_count(current_device());
    if (flash_fits<8, 2, 64>(a) && tall) return flash<8, 2, 64>(a, r, st);
    if (flash_fits<8, 1, 64>(a)) return flash<8, 1, 64>(a, r, st);
    if (flash_fits<16, 2, 64>(a) && tall) return flash<16, 2, 64>(a, r, st);
    if (flash_fits<16, 1, 64>(a)) return flash<16, 1, 64>(a, r, st);
    if (flash_fits<32, 1, 32>(a)) return flash<32, 1, 32>(a, r, st);
    return scalar<bf16>(a, r, st);
}

}  // namespace lm
}  // namespace bw

extern "C" int bw_diff_attention(const bw_diff_attention_args* a, const bw_rows* rows, int f32, void* stream) {
    if (!a || !rows || rows->T < 1 || !a->cs || !a->cache || !a->q || !a->out || (a->k ? !a->v : a->v != nullptr) || a->max_seq < 1 ||
        a->cap < 1 || a->ld % 8 != 0 || a->ldout % 8 != 0 || a->splits < 0 || a->slots < 1 || (rows->row_slot && !rows->row_pos) || rows->pos0 < 0 ||
        (!rows->row_slot && rows->pos0 + rows->T > a->max_seq))
        return cudaErrorInvalidValue;
    const int rows_of_one = rows->row_slot ? 1 : rows->T;
    if (a->cap < a->max_seq && (a->window < 1 || a->cap % 16 != 0 || a->cap < a->window - 1 + rows_of_one)) return cudaErrorInvalidValue;
    bw::lm::DiffAttnArgs d{};
    d.heads = a->heads; d.kv_heads = a->kv_heads; d.dim = a->dim; d.V = a->V; d.window = a->window; d.rot_dims = a->rot_dims;
    d.cs = static_cast<const float2*>(a->cs); d.max_seq = a->max_seq; d.scale = a->scale; d.lambda = a->lambda; d.out_scale = a->out_scale;
    d.eps = a->eps; d.cache = a->cache; d.cap = a->cap; d.slots = a->slots; d.q = a->q; d.k = a->k; d.v = a->v; d.ld = a->ld; d.out = a->out; d.ldout = a->ldout;
    if (!bw::lm::diff_attention_supported(d)) return cudaErrorInvalidValue;
    d.splits = a->splits ? a->splits : bw::lm::diff_attention_splits(d, rows->T, f32);
    const bw::lm::Rows w{rows->T, rows->row_slot, rows->row_pos, rows->slot, rows->pos0};
    return bw::lm::diff_attention(d, w, f32, static_cast<cudaStream_t>(stream));
}
