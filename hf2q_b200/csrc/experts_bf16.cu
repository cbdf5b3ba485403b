// Routed experts with bf16 weights around the grouped products of dense_bf16.cu: choice and grouping of a portion's rows,
// and the two launches that take one token through its experts.
#include "matvec_stream.cuh"

namespace hf2q {
namespace {
using namespace seq;

// sorted row order <- rows of x, 16 bytes per thread and step
__global__ void __launch_bounds__(256) gather_rows_kernel(const uint4* __restrict__ x, uint32_t quads, uint32_t top, const uint32_t* __restrict__ header,
                                                          const uint32_t* __restrict__ perm, uint4* __restrict__ xg) {
    pdl_trigger();
    pdl_wait();
    const uint32_t n = header[1];
    for (uint32_t r = blockIdx.x; r < n; r += gridDim.x) {
        const uint4* src = x + static_cast<size_t>(perm[r] / top) * quads;
        for (uint32_t i = threadIdx.x; i < quads; i += blockDim.x) xg[static_cast<size_t>(r) * quads + i] = src[i];
    }
}

// The `top` largest sigmoid scores by counting, for every expert, those in front of it; z, ids, scores in shared memory.
// An expert id is written for every place whatever the logits hold.
__device__ __forceinline__ void choose_experts(const float* logits, uint32_t experts, uint32_t top, float* z, uint32_t* ids, float* scores) {
    for (uint32_t i = threadIdx.x; i < experts; i += blockDim.x) z[i] = sigmoidf(logits[i]);
    for (uint32_t i = threadIdx.x; i < top; i += blockDim.x) { ids[i] = 0; scores[i] = 0.f; }
    __syncthreads();
    for (uint32_t e = threadIdx.x; e < experts; e += blockDim.x) {
        const float s = z[e];
        uint32_t rank = 0;
        for (uint32_t o = 0; o < experts; ++o) rank += z[o] > s || (z[o] == s && o < e);
        if (rank < top) { ids[rank] = e; scores[rank] = s; }
    }
    __syncthreads();
}

constexpr uint32_t STEP_EXPERTS = 1024, STEP_TOP = 64;

__global__ void __launch_bounds__(MR_THREADS) expert_glu_kernel(const __grid_constant__ hf2q_expert_step e, uint32_t* status) {
    extern __shared__ __align__(128) uint8_t mv_smem[];                 // ring, then h [k_in] f32
    __shared__ MatvecShared sh;
    __shared__ float z[STEP_EXPERTS], scores[STEP_TOP];
    __shared__ uint32_t ids[STEP_TOP];
    pdl_trigger();
    pdl_wait();
    choose_experts(e.logits, e.experts, e.top, z, ids, scores);
    // pairs of rows of all chosen experts, spread evenly
    const uint32_t pairs = e.top * e.ff, per_row = (e.k_in + MV_CHUNK - 1) / MV_CHUNK;
    const uint32_t row0 = 2 * static_cast<uint32_t>(static_cast<uint64_t>(pairs) * blockIdx.x / gridDim.x);
    const uint32_t row1 = 2 * static_cast<uint32_t>(static_cast<uint64_t>(pairs) * (blockIdx.x + 1) / gridDim.x);
    auto chunk = [&](uint32_t c) {
        const uint32_t row = row0 + c / per_row, k0 = (c % per_row) * MV_CHUNK, slot = row / (2 * e.ff);
        const size_t w_row = static_cast<size_t>(ids[slot]) * 2 * e.ff + row % (2 * e.ff);
        return MatvecChunk{static_cast<const __nv_bfloat16*>(e.gate_up) + w_row * e.k_in + k0, k0, min(static_cast<uint32_t>(MV_CHUNK), e.k_in - k0)};
    };
    MatvecStream stream(mv_smem, sh, (row1 - row0) * per_row, status);
    stream.start(chunk);
    float* xs = reinterpret_cast<float*>(mv_smem + MR_RING);
    for (uint32_t i = threadIdx.x; i < e.k_in; i += MR_THREADS) xs[i] = e.h[i];
    if (blockIdx.x == 0)
        for (uint32_t i = threadIdx.x; i < e.top; i += MR_THREADS) e.ids[i] = ids[i];
    __syncthreads();
    stream.run<true>(chunk, xs, row1 - row0, per_row, [&](uint32_t r, float g, float u) {
        const uint32_t row = row0 + r;
        const float s = scores[row / (2 * e.ff)];
        e.act[row / 2] = siluf(s * g) * (s * u);
    });
}

__global__ void __launch_bounds__(MR_THREADS) expert_down_kernel(const __grid_constant__ hf2q_expert_step e, uint32_t* status) {
    extern __shared__ __align__(128) uint8_t mv_smem[];                 // ring, then act [top][ff] f32
    __shared__ MatvecShared sh;
    __shared__ uint32_t ids[STEP_TOP];
    pdl_trigger();
    pdl_wait();
    for (uint32_t i = threadIdx.x; i < e.top; i += MR_THREADS) ids[i] = e.ids[i];
    __syncthreads();
    const uint32_t per_slot = (e.ff + MV_CHUNK - 1) / MV_CHUNK, per_row = e.top * per_slot;
    const uint32_t row0 = static_cast<uint32_t>(static_cast<uint64_t>(e.width) * blockIdx.x / gridDim.x);
    const uint32_t row1 = static_cast<uint32_t>(static_cast<uint64_t>(e.width) * (blockIdx.x + 1) / gridDim.x);
    auto chunk = [&](uint32_t c) {                                      // a row's chunks: expert after expert
        const uint32_t row = row0 + c / per_row, slot = c % per_row / per_slot, k0 = (c % per_slot) * MV_CHUNK;
        const size_t w_row = static_cast<size_t>(ids[slot]) * e.width + row;
        return MatvecChunk{static_cast<const __nv_bfloat16*>(e.down) + w_row * e.ff + k0, slot * e.ff + k0, min(static_cast<uint32_t>(MV_CHUNK), e.ff - k0)};
    };
    MatvecStream stream(mv_smem, sh, (row1 - row0) * per_row, status);
    stream.start(chunk);
    float* xs = reinterpret_cast<float*>(mv_smem + MR_RING);
    for (uint32_t i = threadIdx.x; i < e.top * e.ff; i += MR_THREADS) xs[i] = e.act[i];
    __syncthreads();
    stream.run<false>(chunk, xs, row1 - row0, per_row, [&](uint32_t r, float v, float) { e.y[row0 + r] = v; });
}

constexpr uint32_t STEP_SMEM = 200 * 1024;                              // (the choice needs some static shared memory as well)

bool step_ok(const hf2q_expert_step* e) {
    return e && e->gate_up && e->down && e->logits && e->h && e->ids && e->act && e->y && e->experts && e->experts <= STEP_EXPERTS && e->top && e->top <= STEP_TOP &&
           e->top <= e->experts && e->ff && e->ff % 8 == 0 && e->k_in && e->k_in % 8 == 0 && e->width && MR_RING + e->k_in * 4ull <= STEP_SMEM &&
           MR_RING + 4ull * e->top * e->ff <= STEP_SMEM && e->top * static_cast<uint64_t>((e->ff + MV_CHUNK - 1) / MV_CHUNK) <= MR_PART &&
           (reinterpret_cast<uintptr_t>(e->gate_up) | reinterpret_cast<uintptr_t>(e->down)) % 16 == 0;
}

}  // namespace
}  // namespace hf2q

using namespace hf2q;
using namespace hf2q::seq;

extern "C" {

HF2Q_API int32_t hf2q_cuda_moe_sigmoid_topk(hf2q_ctx* ctx, void* stream, const float* logits, uint32_t ld, uint32_t* ids, float* weights, uint32_t m,
                                            uint32_t experts, uint32_t top) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!logits || !ids || !weights || experts == 0 || ld < experts || top == 0 || top > experts)
        return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "moe_sigmoid_topk: null pointer or a bad size");
    if (m == 0) return HF2Q_OK;
    return ctx_cuda_result(ctx, launch_sigmoid_topk(logits, ld, ids, weights, m, experts, top, static_cast<cudaStream_t>(stream)), "moe_sigmoid_topk", 1);
}

HF2Q_API int32_t hf2q_cuda_sort_rows(hf2q_ctx* ctx, void* stream, const uint32_t* ids, uint32_t m, uint32_t top, uint32_t experts, uint32_t tile_rows,
                                     const void* x, uint32_t dtype, uint32_t ldx, uint32_t* header, void* tiles, uint32_t* perm, void* xg) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!ids || !x || !header || !tiles || !perm || !xg || top == 0 || experts == 0 || tile_rows == 0 || ldx == 0 || ldx % 8 ||
        (dtype != HF2Q_DT_F32 && dtype != HF2Q_DT_BF16) || (reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(xg) | reinterpret_cast<uintptr_t>(tiles)) % 16)
        return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "sort_rows: null or unaligned pointer, or a bad size");
    if (m == 0) return HF2Q_OK;
    const cudaStream_t st = static_cast<cudaStream_t>(stream);
    cudaError_t e = launch_moe_sort(ids, m * top, experts, tile_rows, header, tiles, perm, nullptr, nullptr, 0, ctx_status_word(ctx), st);
    const uint32_t quads = ldx * (dtype == HF2Q_DT_F32 ? 4 : 2) / 16, rows = m * top, cap = static_cast<uint32_t>(ctx_sm_count(ctx)) * 8;
    if (e == cudaSuccess)
        e = launch_pdl(gather_rows_kernel, dim3(rows < cap ? rows : cap), dim3(256), 0, st, static_cast<const uint4*>(x), quads, top, header, perm, static_cast<uint4*>(xg));
    return ctx_cuda_result(ctx, e, "sort_rows", 2);
}

HF2Q_API int32_t hf2q_cuda_expert_glu_step(hf2q_ctx* ctx, void* stream, const hf2q_expert_step* e) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!step_ok(e)) return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "expert_glu_step: null or unaligned pointer, or a size outside the limits");
    static PerDeviceFlag flag;
    cudaError_t r = ensure_max_dynamic_smem(expert_glu_kernel, STEP_SMEM, flag);
    const uint32_t sms = static_cast<uint32_t>(ctx_sm_count(ctx)), pairs = e->top * e->ff;
    if (r == cudaSuccess)
        r = launch_pdl(expert_glu_kernel, dim3(pairs < sms ? pairs : sms), dim3(MR_THREADS), MR_RING + static_cast<size_t>(e->k_in) * 4, static_cast<cudaStream_t>(stream), *e,
                       ctx_status_word(ctx));
    return ctx_cuda_result(ctx, r, "expert_glu_step", 1);
}

HF2Q_API int32_t hf2q_cuda_expert_down_step(hf2q_ctx* ctx, void* stream, const hf2q_expert_step* e) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!step_ok(e)) return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "expert_down_step: null or unaligned pointer, or a size outside the limits");
    static PerDeviceFlag flag;
    cudaError_t r = ensure_max_dynamic_smem(expert_down_kernel, STEP_SMEM, flag);
    const uint32_t sms = static_cast<uint32_t>(ctx_sm_count(ctx));
    if (r == cudaSuccess)
        r = launch_pdl(expert_down_kernel, dim3(e->width < sms ? e->width : sms), dim3(MR_THREADS), MR_RING + 4ull * e->top * e->ff, static_cast<cudaStream_t>(stream), *e,
                       ctx_status_word(ctx));
    return ctx_cuda_result(ctx, r, "expert_down_step", 1);
}

}  // extern "C"
