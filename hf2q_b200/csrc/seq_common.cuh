// Shared device helpers of the bf16-weight sequence-model kernels (dense_bf16.cu, window_attn.cu,
// scan.cu, seq_ops.cu): element conversion, block reductions, programmatic dependent launch, and the
// row prologues that both the stand-alone kernels and the fused mat-vec use.
#pragma once
#include "common.cuh"
#include "kernels.h"

namespace hf2q {
namespace seq {

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float bf_lo(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float bf_hi(uint32_t w) { return __uint_as_float(w & 0xffff0000u); }

// eight consecutive elements (16-byte aligned for bf16, 32 bytes read as two 16-byte loads for f32)
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&o)[8]) {
    const uint4 v = *reinterpret_cast<const uint4*>(p);
    o[0] = bf_lo(v.x); o[1] = bf_hi(v.x); o[2] = bf_lo(v.y); o[3] = bf_hi(v.y);
    o[4] = bf_lo(v.z); o[5] = bf_hi(v.z); o[6] = bf_lo(v.w); o[7] = bf_hi(v.w);
}
__device__ __forceinline__ void load8(const float* p, float (&o)[8]) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    o[0] = a.x; o[1] = a.y; o[2] = a.z; o[3] = a.w; o[4] = b.x; o[5] = b.y; o[6] = b.z; o[7] = b.w;
}

__device__ __forceinline__ float sigmoidf(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplusf(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float siluf(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float gelu_tanhf(float x) {
    return 0.5f * x * (1.0f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x)));
}

// ---- product epilogues that take rows in pairs (gate, up)
__host__ __device__ constexpr bool epi_pairs(uint32_t epi) { return epi == HF2Q_EPI_SWIGLU || epi == HF2Q_EPI_CLAMP_GLU; }
__host__ __device__ constexpr bool epi_needs_cap(uint32_t epi) { return epi == HF2Q_EPI_SOFTCAP || epi == HF2Q_EPI_CLAMP_GLU; }
__device__ __forceinline__ float glu_value(float gate, float up, uint32_t epi, float cap) {
    if (epi == HF2Q_EPI_SWIGLU) return siluf(gate) * up;
    const float g = fminf(gate, cap), u = fminf(fmaxf(up, -cap), cap);
    return g * sigmoidf(1.702f * g) * (u + 1.0f);
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// Sum of N values over the block; red: N * 32 floats of shared memory.  Ends with every thread holding the
// sums; the caller may reuse `red` only after another barrier.
template <int N>
__device__ __forceinline__ void block_sum(float (&v)[N], float* red) {
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] = warp_sum(v[i]);
    if ((threadIdx.x & 31) == 0)
#pragma unroll
        for (int i = 0; i < N; ++i) red[i * 32 + (threadIdx.x >> 5)] = v[i];
    __syncthreads();
    const uint32_t lane = threadIdx.x & 31, nw = blockDim.x >> 5;
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] = warp_sum(lane < nw ? red[i * 32 + lane] : 0.f);
}

// Programmatic dependent launch.  Every kernel launched with launch_pdl() calls pdl_wait() before it touches
// memory that an earlier kernel of the stream writes (or still reads); weights may be touched before.
__device__ __forceinline__ void pdl_trigger() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void prefetch_l2(const void* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }

template <typename... KArgs, typename... Args>
inline cudaError_t launch_pdl(void (*kern)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t st, Args... args) {
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    return cudaLaunchKernelEx(&cfg, kern, static_cast<KArgs>(args)...);
}

template <typename... KArgs, typename... Args>
inline cudaError_t launch_pdl_cluster(void (*kern)(KArgs...), dim3 grid, dim3 block, dim3 cluster, size_t smem, cudaStream_t st, Args... args) {
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = cluster.x;
    attr[1].val.clusterDim.y = cluster.y;
    attr[1].val.clusterDim.z = cluster.z;
    cfg.attrs = attr;
    cfg.numAttrs = 2;
    return cudaLaunchKernelEx(&cfg, kern, static_cast<KArgs>(args)...);
}

__device__ __forceinline__ void cp_async4(void* dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// ---------------------------------------------------------------- row prologues
// rows whose width is a multiple of four are read in 16-byte groups
inline bool pre_norm_aligned(const hf2q_pre_norm& p) {
    if (p.width % 4) return true;
    const void* all[] = {p.x, p.a, p.b, p.a_norm, p.b_norm, p.add0, p.step};
    for (const void* q : all)
        if (reinterpret_cast<uintptr_t>(q) % 16) return false;
    return true;
}

// Residual update of row t into xs[0..width) (shared memory):
//   x + 0.5 (rms(a) a_norm + rms(b) b_norm)  (+ add0)  (+ step)
// and the reciprocal root mean square of the result.  Rows are `width` floats apart.
__device__ __forceinline__ float residual_row(const hf2q_pre_norm& p, uint32_t t, float* xs, float* red) {
    const size_t o = static_cast<size_t>(t) * p.width;
    const float n = static_cast<float>(p.width);
    const bool quads = p.width % 4 == 0;                   // rows of whole 16-byte groups
    const uint32_t nq = quads ? p.width / 4 : 0;
    auto q4 = [](const float* b, uint32_t i) { return *reinterpret_cast<const float4*>(b + 4 * i); };
    float ia = 0.f, ib = 0.f;
    if (p.a) {
        float s[2] = {0.f, 0.f};
        for (uint32_t i = threadIdx.x; i < nq; i += blockDim.x) {
            const float4 va = q4(p.a + o, i), vb = q4(p.b + o, i);
            s[0] += va.x * va.x + va.y * va.y + va.z * va.z + va.w * va.w;
            s[1] += vb.x * vb.x + vb.y * vb.y + vb.z * vb.z + vb.w * vb.w;
        }
        for (uint32_t i = 4 * nq + threadIdx.x; i < p.width; i += blockDim.x) {
            const float va = p.a[o + i], vb = p.b[o + i];
            s[0] += va * va;
            s[1] += vb * vb;
        }
        block_sum(s, red);
        ia = 0.5f / sqrtf(s[0] / n + p.eps);
        ib = 0.5f / sqrtf(s[1] / n + p.eps);
        __syncthreads();
    }
    float s[1] = {0.f};
    for (uint32_t i = threadIdx.x; i < nq; i += blockDim.x) {
        float4 v = q4(p.x + o, i);
        if (p.a) {
            const float4 a = q4(p.a + o, i), an = q4(p.a_norm, i), b = q4(p.b + o, i), bn = q4(p.b_norm, i);
            v.x += a.x * ia * an.x + b.x * ib * bn.x; v.y += a.y * ia * an.y + b.y * ib * bn.y;
            v.z += a.z * ia * an.z + b.z * ib * bn.z; v.w += a.w * ia * an.w + b.w * ib * bn.w;
        }
        if (p.add0) { const float4 a = q4(p.add0 + o, i); v.x += a.x; v.y += a.y; v.z += a.z; v.w += a.w; }
        if (p.step) { const float4 a = q4(p.step, i); v.x += a.x; v.y += a.y; v.z += a.z; v.w += a.w; }
        *reinterpret_cast<float4*>(xs + 4 * i) = v;
        s[0] += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    for (uint32_t i = 4 * nq + threadIdx.x; i < p.width; i += blockDim.x) {
        float v = p.x[o + i];
        if (p.a) v += p.a[o + i] * ia * p.a_norm[i] + p.b[o + i] * ib * p.b_norm[i];
        if (p.add0) v += p.add0[o + i];
        if (p.step) v += p.step[i];
        xs[i] = v;
        s[0] += v * v;
    }
    block_sum(s, red);
    const float inv = 1.0f / sqrtf(s[0] / n + p.eps);
    __syncthreads();
    return inv;
}

// One row of gated head outputs into out[0..heads * head_dim): (norm ? o / rms_head(o) * norm : o) * sigmoid(gate);
// one warp per head.  norm_all: the weight spans all heads, else one head_dim vector is shared.
template <typename OUT>
__device__ __forceinline__ void gated_heads_row(const hf2q_gated_heads& g, uint32_t t, OUT* out, uint32_t warp, uint32_t n_warps) {
    const uint32_t lane = threadIdx.x & 31;
    const float* o = g.o + static_cast<size_t>(t) * g.ldo;
    const float* gate = g.gate + static_cast<size_t>(t) * g.ldg;
    // whole 16-byte groups and at most one per lane: a head stays in registers
    const bool quads = g.head_dim % 4 == 0 && g.head_dim <= 128 &&
                       ((reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(g.norm)) & 15) == 0;
    for (uint32_t h = warp; h < g.heads; h += n_warps) {
        const uint32_t c0 = h * g.head_dim;
        if (quads) {
            const uint32_t i = 4 * lane;
            const bool has = i < g.head_dim;
            const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
            const float4 v = has ? *reinterpret_cast<const float4*>(o + c0 + i) : zero, x = has ? *reinterpret_cast<const float4*>(gate + c0 + i) : zero;
            float4 w = make_float4(1.f, 1.f, 1.f, 1.f);
            if (g.norm) {
                const float inv = 1.0f / sqrtf(warp_sum(v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w) / static_cast<float>(g.head_dim) + g.eps);
                if (has) w = *reinterpret_cast<const float4*>(g.norm + (g.norm_all ? c0 + i : i));
                w = make_float4(w.x * inv, w.y * inv, w.z * inv, w.w * inv);
            }
            if (has) {
                out[c0 + i] = from_f32<OUT>(v.x * w.x * sigmoidf(x.x));
                out[c0 + i + 1] = from_f32<OUT>(v.y * w.y * sigmoidf(x.y));
                out[c0 + i + 2] = from_f32<OUT>(v.z * w.z * sigmoidf(x.z));
                out[c0 + i + 3] = from_f32<OUT>(v.w * w.w * sigmoidf(x.w));
            }
            continue;
        }
        float inv = 1.0f;
        if (g.norm) {
            float s = 0.f;
            for (uint32_t i = lane; i < g.head_dim; i += 32) { const float v = o[c0 + i]; s += v * v; }
            inv = 1.0f / sqrtf(warp_sum(s) / static_cast<float>(g.head_dim) + g.eps);
        }
        for (uint32_t i = lane; i < g.head_dim; i += 32) {
            float v = o[c0 + i];
            if (g.norm) v = v * inv * g.norm[g.norm_all ? c0 + i : i];
            out[c0 + i] = from_f32<OUT>(v * sigmoidf(gate[c0 + i]));
        }
    }
}

// One row of a gated, group-normed output: v = o * silu(gate), every one of `heads` equal groups of `head_dim` elements
// divided by its own root mean square, times norm [heads * head_dim].  buf: f32 row in shared memory; out may be buf.
// The whole block takes part; ends without a barrier.
constexpr uint32_t GROUP_MAX = 512;
template <typename OUT>
__device__ __forceinline__ void silu_group_norm_row(const hf2q_gated_heads& g, uint32_t t, float* buf, OUT* out) {
    __shared__ float sums[GROUP_MAX];
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
    const uint32_t sub = max(1u, n_warps / g.heads), units = g.heads * sub;     // warps that share a group
    const float* o = g.o + static_cast<size_t>(t) * g.ldo;
    const float* gate = g.gate + static_cast<size_t>(t) * g.ldg;
    const bool quads = g.head_dim % 4 == 0 && ((reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(gate)) & 15) == 0;
    for (uint32_t u = warp; u < units; u += n_warps) {
        const uint32_t c0 = u / sub * g.head_dim, part = u % sub;
        float s = 0.f;
        if (quads) {
            for (uint32_t i = 4 * (lane + 32 * part); i < g.head_dim; i += 128 * sub) {
                const float4 a = *reinterpret_cast<const float4*>(o + c0 + i), b = *reinterpret_cast<const float4*>(gate + c0 + i);
                const float4 v = make_float4(a.x * siluf(b.x), a.y * siluf(b.y), a.z * siluf(b.z), a.w * siluf(b.w));
                *reinterpret_cast<float4*>(buf + c0 + i) = v;
                s += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
            }
        } else {
            for (uint32_t i = lane + 32 * part; i < g.head_dim; i += 32 * sub) {
                const float v = o[c0 + i] * siluf(gate[c0 + i]);
                buf[c0 + i] = v;
                s += v * v;
            }
        }
        s = warp_sum(s);
        if (lane == 0) sums[u] = s;
    }
    __syncthreads();
    for (uint32_t u = warp; u < units; u += n_warps) {
        const uint32_t c0 = u / sub * g.head_dim, part = u % sub;
        float s = 0.f;
        for (uint32_t k = 0; k < sub; ++k) s += sums[u / sub * sub + k];
        const float inv = 1.0f / sqrtf(s / static_cast<float>(g.head_dim) + g.eps);
        for (uint32_t i = lane + 32 * part; i < g.head_dim; i += 32 * sub) out[c0 + i] = from_f32<OUT>(buf[c0 + i] * inv * g.norm[c0 + i]);
    }
}
inline bool gated_ok(const hf2q_gated_heads& g) {
    return g.o && g.gate && g.heads && g.head_dim && g.kind <= HF2Q_GATE_SILU_FIRST && (g.kind == HF2Q_GATE_SIGMOID_LAST || (g.norm && g.heads <= GROUP_MAX));
}

// ---- several residual streams
constexpr uint32_t HYPER_MAX = 16, HYPER_COEF = HYPER_MAX * HYPER_MAX + 2 * HYPER_MAX;

inline bool hyper_ok(const hf2q_hyper& p) {
    if (!p.x || !p.streams || p.streams > HYPER_MAX || (p.x_streams != 1 && p.x_streams != p.streams) || !p.width || (p.y && (!p.mix || !p.out || !p.y_parts)) ||
        (p.x_out == p.x && p.x_streams != p.streams))
        return false;
    if (p.width % 4) return true;
    const void* all[] = {p.x, p.x_out, p.y};
    for (const void* q : all)
        if (reinterpret_cast<uintptr_t>(q) % 16) return false;
    return true;
}

// V: float or float4 (width a multiple of four)
__device__ __forceinline__ void axpy(float& d, float a, float x) { d = fmaf(a, x, d); }
__device__ __forceinline__ void axpy(float4& d, float a, const float4& x) { d.x = fmaf(a, x.x, d.x); d.y = fmaf(a, x.y, d.y); d.z = fmaf(a, x.z, d.z); d.w = fmaf(a, x.w, d.w); }
__device__ __forceinline__ float square_sum(float v) { return v * v; }
__device__ __forceinline__ float square_sum(const float4& v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }

template <int S, typename V>
__device__ __forceinline__ float hyper_elements(const hf2q_hyper& p, uint32_t t, float* xs, const float* coef, uint32_t lo, uint32_t hi) {
    constexpr uint32_t E = sizeof(V) / 4;
    const uint32_t n = p.width / E;
    const V* x = reinterpret_cast<const V*>(p.x + static_cast<size_t>(t) * p.x_streams * p.width);
    V* xo = reinterpret_cast<V*>(p.x_out + static_cast<size_t>(t) * p.streams * p.width);
    const V* y = reinterpret_cast<const V*>(p.y + static_cast<size_t>(t) * p.y_parts * p.width);
    const float *mix = coef, *out = coef + S * S, *in = out + S;
    float ss = 0.f;
    for (uint32_t i = threadIdx.x; i < n; i += blockDim.x) {
        V old[S], yv{}, u{};
#pragma unroll
        for (int s = 0; s < S; ++s) old[s] = s < static_cast<int>(p.streams) ? x[(p.x_streams == 1 ? 0u : s * n) + i] : V{};
        if (p.y)
            for (uint32_t k = 0; k < p.y_parts; ++k) axpy(yv, 1.0f, y[k * n + i]);
        const bool own = p.x_out && E * i >= lo && E * i < hi;
#pragma unroll
        for (int d = 0; d < S; ++d) {
            if (d >= static_cast<int>(p.streams)) continue;
            V v = old[d];
            if (p.y) {
                v = V{};
#pragma unroll
                for (int s = 0; s < S; ++s) axpy(v, mix[s * S + d], old[s]);
                axpy(v, out[d], yv);
            }
            if (own) xo[d * n + i] = v;
            axpy(u, in[d], v);
        }
        reinterpret_cast<V*>(xs)[i] = u;
        ss += square_sum(u);
    }
    return ss;
}
template <int S>
__device__ __forceinline__ float hyper_row_s(const hf2q_hyper& p, uint32_t t, float* xs, float* coef, uint32_t lo, uint32_t hi) {
    // [S][S] mix, [S] out, [S] in; absent streams have zeros
    for (uint32_t i = threadIdx.x; i < S * S + 2 * S; i += blockDim.x) {
        const uint32_t a = i / S, b = i % S;
        float v = 0.f;
        if (b < p.streams) {
            if (a < S) v = p.y && a < p.streams ? p.mix[a * p.streams + b] : 0.f;
            else if (a == S) v = p.y ? p.out[b] : 0.f;
            else v = p.in ? p.in[b] : 1.0f;
        }
        coef[i] = v;
    }
    __syncthreads();
    return p.width % 4 == 0 ? hyper_elements<S, float4>(p, t, xs, coef, lo, hi) : hyper_elements<S, float>(p, t, xs, coef, lo, hi);
}
// Row t of the streams (hf2q_hyper): the pending update, stored for elements [lo, hi), and the row that the sublayer reads
// into xs[0..width) (shared memory, 16-byte aligned).  Returns the reciprocal root mean square of it.
__device__ __forceinline__ float hyper_row(const hf2q_hyper& p, uint32_t t, float* xs, float* coef, float* red, uint32_t lo, uint32_t hi) {
    float s[1];
    if (p.streams <= 2) s[0] = hyper_row_s<2>(p, t, xs, coef, lo, hi);
    else if (p.streams <= 4) s[0] = hyper_row_s<4>(p, t, xs, coef, lo, hi);
    else if (p.streams <= 8) s[0] = hyper_row_s<8>(p, t, xs, coef, lo, hi);
    else s[0] = hyper_row_s<16>(p, t, xs, coef, lo, hi);
    block_sum(s, red);
    return 1.0f / sqrtf(s[0] / static_cast<float>(p.width) + p.eps);
}

}  // namespace seq
}  // namespace hf2q
