// Row-wise steps around the products of a bf16-weight decoder: embedding rows with the hashed bigram table, the
// residual update + RMS norm + token shift in front of a product, the same for a residual in several streams, gated head outputs, and the hand-over of the
// shift / convolution state after a portion of several tokens.
#include "seq_common.cuh"

namespace hf2q {
namespace {
using namespace seq;

__global__ void __launch_bounds__(256) embed_kernel(const __grid_constant__ hf2q_embed e, const uint32_t* __restrict__ ids, uint32_t m,
                                                    float* __restrict__ x, uint32_t* status) {
    pdl_trigger();
    pdl_wait();
    const uint32_t t = blockIdx.x;
    const uint32_t id = ids[t], pos = *e.pos + t;
    const uint32_t before = t ? ids[t - 1] : *e.prev;
    const uint32_t last = ids[m - 1];
    __syncthreads();                                       // row 0 reads *prev before it replaces it
    if (t == 0 && threadIdx.x == 0) *e.prev = last;
    const bool bad = id >= e.vocab;
    if (bad && threadIdx.x == 0) atomicOr(status, STATUS_BAD_EXPERT_ID);
    const __nv_bfloat16* row = static_cast<const __nv_bfloat16*>(e.embed) + static_cast<size_t>(bad ? 0 : id) * e.ld;
    const __nv_bfloat16* big = nullptr;
    if (e.bigram) {
        const uint64_t r = pos == 0 ? e.buckets : (before * e.mul_prev + id * e.mul_cur) % e.buckets;
        big = static_cast<const __nv_bfloat16*>(e.bigram) + r * e.ld;
    }
    for (uint32_t i = threadIdx.x; i < e.width; i += blockDim.x) {
        float v = bad ? 0.f : to_f32(row[i]);
        if (big) v += to_f32(big[i]);
        x[static_cast<size_t>(t) * e.width + i] = v;
    }
}

// `run` consecutive rows per CTA; a token shift needs the row before the first as well, recomputed from the same inputs
template <typename OUT>
__global__ void __launch_bounds__(512) pre_norm_kernel(const __grid_constant__ hf2q_pre_norm p, uint32_t m, uint32_t run, OUT* __restrict__ out, uint32_t ldo,
                                                       float* __restrict__ h_last) {
    extern __shared__ __align__(16) float xs[];            // width, and another width with a shift: the h of the row before
    __shared__ float red[64];
    pdl_trigger();
    pdl_wait();
    const uint32_t t0 = blockIdx.x * run, t1 = min(t0 + run, m);
    const uint32_t pos = p.shift ? *p.pos : 0u;
    float* before = xs + p.width;                          // an element is read and written by one thread only
    if (p.shift) {
        if (t0 > 0) {
            const float inv = residual_row(p, t0 - 1, before, red);
            for (uint32_t i = threadIdx.x; i < p.width; i += blockDim.x) before[i] *= inv * p.norm[i];
        } else {
            for (uint32_t i = threadIdx.x; i < p.width; i += blockDim.x) before[i] = p.shift_state[static_cast<size_t>((pos + 1) & 1) * p.width + i];
        }
    }
    const bool quads = p.width % 4 == 0 && ldo == p.width &&
                       ((reinterpret_cast<uintptr_t>(p.norm) | reinterpret_cast<uintptr_t>(p.shift) | reinterpret_cast<uintptr_t>(p.x_out) |
                         reinterpret_cast<uintptr_t>(p.shift_state) | reinterpret_cast<uintptr_t>(h_last) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
    if (quads) __syncthreads();                            // `before` changes hands: groups of four per thread from here on
    for (uint32_t t = t0; t < t1; ++t) {
        const float inv = residual_row(p, t, xs, red);
        if (quads) {
            for (uint32_t i = threadIdx.x; i < p.width / 4; i += blockDim.x) {
                const float4 x = reinterpret_cast<const float4*>(xs)[i], w = reinterpret_cast<const float4*>(p.norm)[i];
                if (p.x_out) reinterpret_cast<float4*>(p.x_out + static_cast<size_t>(t) * p.width)[i] = x;
                float4 h = make_float4(x.x * inv * w.x, x.y * inv * w.y, x.z * inv * w.z, x.w * inv * w.w);
                if (p.shift) {
                    const float4 b = reinterpret_cast<const float4*>(before)[i], mu = reinterpret_cast<const float4*>(p.shift)[i];
                    reinterpret_cast<float4*>(before)[i] = h;
                    if (m == 1) reinterpret_cast<float4*>(p.shift_state + static_cast<size_t>(pos & 1) * p.width)[i] = h;
                    else if (t == m - 1) reinterpret_cast<float4*>(h_last)[i] = h;
                    h = make_float4(h.x + (b.x - h.x) * mu.x, h.y + (b.y - h.y) * mu.y, h.z + (b.z - h.z) * mu.z, h.w + (b.w - h.w) * mu.w);
                }
                OUT* dst = out + static_cast<size_t>(t) * ldo + 4 * i;
                if constexpr (sizeof(OUT) == 4) {
                    *reinterpret_cast<float4*>(dst) = h;
                } else {
                    const __nv_bfloat162 lo = __floats2bfloat162_rn(h.x, h.y), hi = __floats2bfloat162_rn(h.z, h.w);
                    *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
                }
            }
            __syncthreads();
            continue;
        }
        for (uint32_t i = threadIdx.x; i < ldo; i += blockDim.x) {
            float h = 0.f;
            if (i < p.width) {
                const float x = xs[i];
                if (p.x_out) p.x_out[static_cast<size_t>(t) * p.width + i] = x;
                h = x * inv * p.norm[i];
                if (p.shift) {
                    const float b = before[i];
                    before[i] = h;
                    if (m == 1) p.shift_state[static_cast<size_t>(pos & 1) * p.width + i] = h;
                    else if (t == m - 1) h_last[i] = h;
                    h += (b - h) * p.shift[i];
                }
            }
            out[static_cast<size_t>(t) * ldo + i] = from_f32<OUT>(h);
        }
        __syncthreads();                                   // xs is read across threads before the next row replaces it
    }
}

template <typename OUT>
__global__ void __launch_bounds__(512) hyper_norm_kernel(const __grid_constant__ hf2q_hyper p, OUT* __restrict__ out, uint32_t ldo) {
    extern __shared__ __align__(16) float xs[];
    __shared__ float coef[HYPER_COEF];
    __shared__ float red[32];
    pdl_trigger();
    pdl_wait();
    const uint32_t t = blockIdx.x;
    const float inv = hyper_row(p, t, xs, coef, red, 0, p.width);
    OUT* row = out + static_cast<size_t>(t) * ldo;
    if (p.width % 4 == 0 && ldo % 4 == 0 && ((reinterpret_cast<uintptr_t>(p.norm) | reinterpret_cast<uintptr_t>(out)) & 15) == 0) {
        for (uint32_t i = threadIdx.x; i < ldo / 4; i += blockDim.x) {
            float4 h = make_float4(0.f, 0.f, 0.f, 0.f);
            if (4 * i < p.width) {
                h = reinterpret_cast<const float4*>(xs)[i];
                if (p.norm) {
                    const float4 w = reinterpret_cast<const float4*>(p.norm)[i];
                    h = make_float4(h.x * inv * w.x, h.y * inv * w.y, h.z * inv * w.z, h.w * inv * w.w);
                }
            }
            if constexpr (sizeof(OUT) == 4) {
                reinterpret_cast<float4*>(row)[i] = h;
            } else {
                const __nv_bfloat162 a = __floats2bfloat162_rn(h.x, h.y), b = __floats2bfloat162_rn(h.z, h.w);
                reinterpret_cast<uint2*>(row)[i] = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
            }
        }
        return;
    }
    for (uint32_t i = threadIdx.x; i < ldo; i += blockDim.x)
        row[i] = from_f32<OUT>(i < p.width ? (p.norm ? xs[i] * inv * p.norm[i] : xs[i]) : 0.f);
}

template <typename OUT>
__global__ void __launch_bounds__(256) gated_heads_kernel(const __grid_constant__ hf2q_gated_heads g, OUT* __restrict__ out, uint32_t ldo) {
    pdl_trigger();
    pdl_wait();
    const uint32_t t = blockIdx.x;
    OUT* row = out + static_cast<size_t>(t) * ldo;
    for (uint32_t i = g.heads * g.head_dim + threadIdx.x; i < ldo; i += blockDim.x) row[i] = from_f32<OUT>(0.f);
    extern __shared__ __align__(16) float buf[];
    if (g.kind == HF2Q_GATE_SILU_FIRST) silu_group_norm_row<OUT>(g, t, buf, row);
    else gated_heads_row<OUT>(g, t, row, threadIdx.x >> 5, blockDim.x >> 5);
}

__global__ void __launch_bounds__(256) state_tail_kernel(const uint32_t* __restrict__ pos_dev, uint32_t m, const float* __restrict__ h_last,
                                                         float* __restrict__ shift_state, uint32_t width, const __grid_constant__ hf2q_delta d,
                                                         uint32_t channels) {
    pdl_trigger();
    pdl_wait();
    const uint32_t pos = *pos_dev;
    const uint32_t i = blockIdx.x * blockDim.x + threadIdx.x;
    if (shift_state && i < width) shift_state[static_cast<size_t>((pos + m - 1) & 1) * width + i] = h_last[i];
    if (i < channels) {
        // inputs of the last taps - 1 positions; those before this portion are in the state already
        const uint32_t qk = d.kv_heads * d.dim;
        const uint32_t col = i < qk ? d.q_off + i : i < 2 * qk ? d.k_off + (i - qk) : d.v_off + (i - 2 * qk);
        const uint32_t keep = d.taps - 1 < m ? d.taps - 1 : m;
        for (uint32_t j = 0; j < keep; ++j) {
            const uint32_t t = m - 1 - j;
            d.conv_state[static_cast<size_t>(i) * d.taps + (pos + t) % d.taps] = d.proj[static_cast<size_t>(t) * d.ld + col];
        }
    }
}

}  // namespace
}  // namespace hf2q

using namespace hf2q;
using namespace hf2q::seq;

extern "C" {

HF2Q_API int32_t hf2q_cuda_embed(hf2q_ctx* ctx, void* stream, const hf2q_embed* e, const uint32_t* ids, uint32_t m, float* x) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!e || !e->embed || !e->pos || !e->prev || !ids || !x || e->vocab == 0 || e->width == 0 || e->ld < e->width || (e->bigram && e->buckets == 0))
        return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "embed: null pointer or empty table");
    if (m == 0) return HF2Q_OK;
    const cudaError_t r = launch_pdl(embed_kernel, dim3(m), dim3(256), 0, static_cast<cudaStream_t>(stream), *e, ids, m, x, ctx_status_word(ctx));
    return ctx_cuda_result(ctx, r, "embed", 1);
}

HF2Q_API int32_t hf2q_cuda_pre_norm(hf2q_ctx* ctx, void* stream, const hf2q_pre_norm* p, uint32_t m, void* out, uint32_t out_dtype, uint32_t ldo,
                                    float* h_last) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!p || !p->x || !p->norm || !out || p->width == 0 || ldo < p->width || p->x_out == p->x || (p->a && (!p->b || !p->a_norm || !p->b_norm)) ||
        (p->shift && (!p->shift_state || !p->pos || (m > 1 && !h_last))) || !pre_norm_aligned(*p))
        return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "pre_norm: null or unaligned pointer, or x_out is x");
    if (m == 0) return HF2Q_OK;
    const size_t smem = static_cast<size_t>(p->width) * (p->shift ? 8 : 4);
    if (smem > 200 * 1024) return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "pre_norm: width too large");
    const cudaStream_t st = static_cast<cudaStream_t>(stream);
    static PerDeviceFlag f32f, bff;
    // long portions: a few rows per CTA while every SM keeps several CTAs
    const uint32_t run = p->shift && m >= 4u * 4u * static_cast<uint32_t>(ctx_sm_count(ctx)) ? 8 : p->shift && m >= 512 ? 4 : 1;
    const dim3 grid((m + run - 1) / run), block(p->width >= 2048 ? 512 : 256);
    cudaError_t e;
    if (out_dtype == HF2Q_DT_F32) {
        e = ensure_max_dynamic_smem(pre_norm_kernel<float>, 200 * 1024, f32f);
        if (e == cudaSuccess) e = launch_pdl(pre_norm_kernel<float>, grid, block, smem, st, *p, m, run, static_cast<float*>(out), ldo, h_last);
    } else if (out_dtype == HF2Q_DT_BF16) {
        e = ensure_max_dynamic_smem(pre_norm_kernel<__nv_bfloat16>, 200 * 1024, bff);
        if (e == cudaSuccess) e = launch_pdl(pre_norm_kernel<__nv_bfloat16>, grid, block, smem, st, *p, m, run, static_cast<__nv_bfloat16*>(out), ldo, h_last);
    } else {
        e = cudaErrorInvalidValue;
    }
    return ctx_cuda_result(ctx, e, "pre_norm", 1);
}

HF2Q_API int32_t hf2q_cuda_gated_heads(hf2q_ctx* ctx, void* stream, const hf2q_gated_heads* g, uint32_t m, void* out, uint32_t out_dtype, uint32_t ldo) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!g || !gated_ok(*g) || !out || ldo < g->heads * g->head_dim) return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "gated_heads: null pointer or a short row");
    if (m == 0) return HF2Q_OK;
    const cudaStream_t st = static_cast<cudaStream_t>(stream);
    const size_t smem = g->kind == HF2Q_GATE_SILU_FIRST ? static_cast<size_t>(g->heads) * g->head_dim * 4 : 0;
    if (smem > 200 * 1024) return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "gated_heads: row too long");
    static PerDeviceFlag f32f, bff;
    cudaError_t e = cudaErrorInvalidValue;
    if (out_dtype == HF2Q_DT_F32) {
        e = ensure_max_dynamic_smem(gated_heads_kernel<float>, 200 * 1024, f32f);
        if (e == cudaSuccess) e = launch_pdl(gated_heads_kernel<float>, dim3(m), dim3(256), smem, st, *g, static_cast<float*>(out), ldo);
    } else if (out_dtype == HF2Q_DT_BF16) {
        e = ensure_max_dynamic_smem(gated_heads_kernel<__nv_bfloat16>, 200 * 1024, bff);
        if (e == cudaSuccess) e = launch_pdl(gated_heads_kernel<__nv_bfloat16>, dim3(m), dim3(256), smem, st, *g, static_cast<__nv_bfloat16*>(out), ldo);
    }
    return ctx_cuda_result(ctx, e, "gated_heads", 1);
}

HF2Q_API int32_t hf2q_cuda_hyper_norm(hf2q_ctx* ctx, void* stream, const hf2q_hyper* p, uint32_t m, void* out, uint32_t out_dtype, uint32_t ldo) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!p || !hyper_ok(*p) || !out || ldo < p->width) return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "hyper_norm: null or unaligned pointer, a bad number of streams or a short row");
    if (m == 0) return HF2Q_OK;
    const size_t smem = static_cast<size_t>(p->width) * 4;
    if (smem > 200 * 1024) return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "hyper_norm: width too large");
    const cudaStream_t st = static_cast<cudaStream_t>(stream);
    const dim3 block(p->width >= 2048 ? 512 : 256);
    static PerDeviceFlag f32f, bff;
    cudaError_t e = cudaErrorInvalidValue;
    if (out_dtype == HF2Q_DT_F32) {
        e = ensure_max_dynamic_smem(hyper_norm_kernel<float>, 200 * 1024, f32f);
        if (e == cudaSuccess) e = launch_pdl(hyper_norm_kernel<float>, dim3(m), block, smem, st, *p, static_cast<float*>(out), ldo);
    } else if (out_dtype == HF2Q_DT_BF16) {
        e = ensure_max_dynamic_smem(hyper_norm_kernel<__nv_bfloat16>, 200 * 1024, bff);
        if (e == cudaSuccess) e = launch_pdl(hyper_norm_kernel<__nv_bfloat16>, dim3(m), block, smem, st, *p, static_cast<__nv_bfloat16*>(out), ldo);
    }
    return ctx_cuda_result(ctx, e, "hyper_norm", 1);
}

HF2Q_API int32_t hf2q_cuda_state_tail(hf2q_ctx* ctx, void* stream, const uint32_t* pos, uint32_t m, const float* h_last, float* shift_state,
                                      uint32_t width, const hf2q_delta* delta) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!pos || m == 0 || (shift_state && !h_last) || (delta && (!delta->proj || !delta->conv_state || delta->taps == 0)))
        return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "state_tail: null pointer");
    const uint32_t channels = delta && delta->taps > 1 ? 2 * delta->kv_heads * delta->dim + delta->heads * delta->vdim : 0;
    const uint32_t n = shift_state && width > channels ? width : channels;
    if (n == 0) return HF2Q_OK;
    const hf2q_delta none{};
    const cudaError_t e = launch_pdl(state_tail_kernel, dim3((n + 255) / 256), dim3(256), 0, static_cast<cudaStream_t>(stream), pos, m, h_last,
                                     shift_state, width, delta ? *delta : none, channels);
    return ctx_cuda_result(ctx, e, "state_tail", 1);
}

}  // extern "C"
