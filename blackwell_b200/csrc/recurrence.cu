// Launchers of the gated linear recurrence.
#include <cuda_runtime.h>

#include <mutex>

#include "../../include/blackwell_b200.h"
#include "host_util.h"
#include "delta_rule.cuh"
#include "recurrence.cuh"

namespace bw {
namespace lm {
namespace {

template <typename A, int NR, bool CONV>
cudaError_t step_inst(const RecurrenceArgs& a, const ConvArgs& c, const Rows& r, cudaStream_t st) {
    const dim3 grid((pad8(a.V) + kRecV - 1) / kRecV, a.heads, r.row_slot ? r.T : 1);
    const int smem = (64 * NR + kRecV + (a.delta ? 4 : 2) * 8 * kRecV) * 4;
    count_launch(1);
    return a.delta ? launch_pdl(recurrence_step_kernel<A, NR, CONV, true>, grid, dim3(kRecThreads), smem, st, a, c, r)
                   : launch_pdl(recurrence_step_kernel<A, NR, CONV, false>, grid, dim3(kRecThreads), smem, st, a, c, r);
}
template <typename A, bool CONV>
cudaError_t step_nr(const RecurrenceArgs& a, const ConvArgs& c, const Rows& r, cudaStream_t st) {
    const int nr = (a.N + 31) / 32;
    return nr <= 1 ? step_inst<A, 1, CONV>(a, c, r, st) : nr <= 2 ? step_inst<A, 2, CONV>(a, c, r, st)
         : nr <= 4 ? step_inst<A, 4, CONV>(a, c, r, st) : nr <= 8 ? step_inst<A, 8, CONV>(a, c, r, st)
         : nr <= 16 ? step_inst<A, 16, CONV>(a, c, r, st) : cudaErrorInvalidValue;
}

template <int NTW, int VT>
cudaError_t chunk_inst(const RecurrenceArgs& a, const Rows& r, cudaStream_t st) {
    static std::once_flag once[kMaxDevices];
    auto kern = recurrence_chunk_kernel<NTW, VT>;
    cudaError_t e = cudaSuccess;
    std::call_once(once[current_device()], [&] {
        e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxDynSmem);
    });
    if (e != cudaSuccess) return e;
    const int nbuf = ChunkSmem(a.N, VT, 2).total <= kMaxDynSmem ? 2 : 1;
    count_launch(1);
    return launch_pdl(kern, dim3((pad8(a.V) + VT - 1) / VT, a.heads), dim3(256), ChunkSmem(a.N, VT, nbuf).total, st, a, r, nbuf);
}

template <int NTW, int VT>
cudaError_t delta_inst(const RecurrenceArgs& a, const Rows& r, cudaStream_t st) {
    static std::once_flag once[kMaxDevices];
    auto kern = delta_chunk_kernel<NTW, VT>;
    cudaError_t e = cudaSuccess;
    std::call_once(once[current_device()], [&] {
        e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxDynSmem);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_prepare_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxDynSmem);
    });
    if (e != cudaSuccess) return e;
    count_launch(2);
    e = launch_pdl(delta_prepare_kernel, dim3(a.heads, (r.T + kChunk - 1) / kChunk), dim3(256), delta_prepare_smem(a.N), st, a, r);
    if (e != cudaSuccess) return e;
    const int nbuf = DeltaSmem(a.N, VT, 2).total <= kMaxDynSmem ? 2 : 1;
    return launch_pdl(kern, dim3((pad8(a.V) + VT - 1) / VT, a.heads), dim3(256), DeltaSmem(a.N, VT, nbuf).total, st, a, r, nbuf);
}

}  // namespace

cudaError_t recurrence_step(const RecurrenceArgs& a, const ConvArgs* conv, const Rows& r, int f32, cudaStream_t st) {
    if (a.groups < 1 || a.heads % a.groups != 0 || (conv && !r.row_slot)) return cudaErrorInvalidValue;
    const ConvArgs none{};
    if (conv) return f32 ? step_nr<float, true>(a, *conv, r, st) : step_nr<bf16, true>(a, *conv, r, st);
    return f32 ? step_nr<float, false>(a, none, r, st) : step_nr<bf16, false>(a, none, r, st);
}

bool recurrence_chunk_supported(const RecurrenceArgs& a) { return a.N <= 256 && ChunkSmem(a.N, 32, 1).total <= kMaxDynSmem; }

cudaError_t recurrence_chunk(const RecurrenceArgs& a, const Rows& r, cudaStream_t st) {
    if (a.groups < 1 || a.heads % a.groups != 0 || r.row_slot || a.delta || !recurrence_chunk_supported(a)) return cudaErrorInvalidValue;
    // narrow state tiles while the wide ones leave SMs idle or two narrow CTAs share an SM
    const int wide = (pad8(a.V) + 63) / 64 * a.heads, sms = sm_count(current_device());
    const bool pairs = ChunkSmem(a.N, 32, 2).total <= 112 * 1024;
    const bool narrow = a.V <= 32 || wide <= (pairs ? sms : sms / 2) || ChunkSmem(a.N, 64, 1).total > kMaxDynSmem;
    if (pad16(a.N) <= 128) return narrow ? chunk_inst<1, 32>(a, r, st) : chunk_inst<1, 64>(a, r, st);
    return narrow ? chunk_inst<2, 32>(a, r, st) : chunk_inst<2, 64>(a, r, st);
}

size_t delta_chunk_bytes(int rows, int heads) { return (size_t)((rows + kChunk - 1) / kChunk) * heads * kDeltaUnit; }

bool delta_chunk_supported(const RecurrenceArgs& a) { return a.N <= 256 && DeltaSmem(a.N, 32, 1).total <= kMaxDynSmem; }

cudaError_t delta_chunk(const RecurrenceArgs& a, const Rows& r, cudaStream_t st) {
    if (a.groups < 1 || a.heads % a.groups != 0 || r.row_slot || !a.delta || !a.chunk_scratch || !a.log_decay || !a.weight ||
        !delta_chunk_supported(a))
        return cudaErrorInvalidValue;
    // wide state tiles only where the narrow ones need more than one round of CTAs
    const int sms = sm_count(current_device()), narrow = (pad8(a.V) + 31) / 32 * a.heads;
    const bool wide = a.V > 32 && narrow > sms && DeltaSmem(a.N, 64, 1).total <= kMaxDynSmem;
    if (pad16(a.N) <= 128) return wide ? delta_inst<1, 64>(a, r, st) : delta_inst<1, 32>(a, r, st);
    return wide ? delta_inst<2, 64>(a, r, st) : delta_inst<2, 32>(a, r, st);
}

}  // namespace lm
}  // namespace bw

namespace {

bool recurrence_args(const bw_recurrence_args* a, const bw_rows* rows, bw::lm::RecurrenceArgs* r, bw::lm::Rows* w) {
    if (!a || !rows || rows->T < 1 || !a->q || !a->k || !a->v || !a->S || !a->o || a->heads < 1 || a->N < 1 || a->V < 1 ||
        a->groups < 1 || (a->log_decay ? !a->weight : !a->head_log_decay) || (rows->row_slot && !rows->row_pos) ||
        a->ldq % 8 != 0 || a->ldk % 8 != 0 || a->ldv % 8 != 0 || a->ldo % 8 != 0)
        return false;
    r->q = a->q; r->k = a->k; r->v = a->v; r->ldq = a->ldq; r->ldk = a->ldk; r->ldv = a->ldv; r->heads = a->heads; r->N = a->N; r->V = a->V;
    r->groups = a->groups; r->log_decay = a->log_decay; r->weight = a->weight; r->head_log_decay = a->head_log_decay;
    r->const_weight = a->const_weight; r->D = a->D; r->S = a->S; r->o = a->o; r->ldo = a->ldo;
    *w = bw::lm::Rows{rows->T, rows->row_slot, rows->row_pos, rows->slot, rows->pos0};
    return true;
}

}  // namespace

extern "C" int bw_linear_recurrence(const bw_recurrence_args* a, const bw_rows* rows, int chunked, int f32, void* stream) {
    bw::lm::RecurrenceArgs r{};
    bw::lm::Rows w{};
    if (!recurrence_args(a, rows, &r, &w)) return cudaErrorInvalidValue;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (chunked) return f32 ? cudaErrorInvalidValue : bw::lm::recurrence_chunk(r, w, st);
    return bw::lm::recurrence_step(r, nullptr, w, f32, st);
}

extern "C" size_t bw_delta_rule_scratch_bytes(int rows, int heads) { return rows > 0 && heads > 0 ? bw::lm::delta_chunk_bytes(rows, heads) : 0; }

extern "C" int bw_delta_rule(const bw_recurrence_args* a, float unit_eps, float q_scale, void* scratch, const bw_rows* rows, int chunked,
                             int f32, void* stream) {
    bw::lm::RecurrenceArgs r{};
    bw::lm::Rows w{};
    if (!recurrence_args(a, rows, &r, &w) || !r.log_decay || r.D) return cudaErrorInvalidValue;
    r.delta = 1; r.unit_eps = unit_eps; r.q_scale = q_scale; r.chunk_scratch = scratch;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (chunked) return f32 ? cudaErrorInvalidValue : bw::lm::delta_chunk(r, w, st);
    return bw::lm::recurrence_step(r, nullptr, w, f32, st);
}
