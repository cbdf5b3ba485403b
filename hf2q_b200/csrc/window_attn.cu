// Sliding-window attention over a ring cache (position p in slot p % capacity) with grouped query heads, optional
// per-head RMS norm of q and k and an optional logarithmic distance term taken off the scores.  The prefill also runs over
// plain rows of keys and values, with a part of every key shared by the heads (expanded latents).
//
//   append    prefill: normalised queries to a buffer, normalised keys and values to the cache
//   prefill   bf16 cache: tiles of 64 queries x 64 keys on the tensor cores (f32 scores, softmax and accumulators, bf16
//             product operands); f32 cache: one warp per query in f32
//   decode    one launch: norm, append, window split over CTAs, merge by the CTA that arrives last
#include <math_constants.h>

#include "mma_sync.cuh"
#include "seq_common.cuh"

namespace hf2q {
namespace {
using namespace seq;

__host__ __device__ constexpr uint32_t pad8(uint32_t n) { return (n + 7) & ~7u; }

// q . k * scale - r1 ln(1 + r2 distance)
__device__ __forceinline__ float score_of(float dot, float scale, float r1, float r2, uint32_t dist, bool bias) {
    float s = dot * scale;
    if (bias) s -= r1 * logf(1.0f + r2 * static_cast<float>(dist));
    return s;
}

// where a KV head's keys and values are: rings, or with PLAIN rows that start at position `first` and a shared key part
template <typename T, bool PLAIN>
struct KeyRows {
    const T *k, *v, *shared;
    uint32_t capacity, dp, sp, k_row, v_row, first, s_row, s_capacity;      // sp: padded size of the shared part
    __device__ __forceinline__ KeyRows(const hf2q_window_attn& a, uint32_t kvh, uint32_t pos0) {
        const uint32_t dvp = pad8(a.vdim);
        dp = pad8(a.dim);
        capacity = a.capacity;
        if constexpr (PLAIN) {
            sp = pad8(a.shared_dim);
            k_row = v_row = a.row_stride;
            first = pos0 + 1 > a.window ? pos0 + 1 - a.window : 0u;
            k = static_cast<const T*>(a.k_cache) + static_cast<size_t>(kvh) * a.k_head_stride;
            v = static_cast<const T*>(a.v_cache) + static_cast<size_t>(kvh) * a.v_head_stride;
            shared = static_cast<const T*>(a.k_shared);
            s_row = a.shared_stride;
            s_capacity = a.shared_capacity;
        } else {
            sp = 0;
            k_row = dp;
            v_row = dvp;
            k = static_cast<const T*>(a.k_cache) + static_cast<size_t>(kvh) * a.capacity * dp;
            v = static_cast<const T*>(a.v_cache) + static_cast<size_t>(kvh) * a.capacity * dvp;
        }
    }
    __device__ __forceinline__ uint32_t slot(uint32_t p) const {
        if constexpr (PLAIN) return p - first;
        else return p % capacity;
    }
    __device__ __forceinline__ const T* key(uint32_t p) const { return k + static_cast<size_t>(slot(p)) * k_row; }
    __device__ __forceinline__ const T* value(uint32_t p) const { return v + static_cast<size_t>(slot(p)) * v_row; }
    __device__ __forceinline__ const T* shared_key(uint32_t p) const { return shared + static_cast<size_t>(p % s_capacity) * s_row; }
};

// one head vector of up to 256 elements held by a warp (element lane + 32 j), divided by its root mean square
struct HeadVec {
    float v[8];
    __device__ __forceinline__ void load(const float* p, uint32_t dim, uint32_t lane) {
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = lane + 32 * j < dim ? p[lane + 32 * j] : 0.f;
    }
    __device__ __forceinline__ void norm(const float* w, float eps, uint32_t dim, uint32_t lane) {
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) s += v[j] * v[j];
        const float inv = 1.0f / sqrtf(warp_sum(s) / static_cast<float>(dim) + eps);
#pragma unroll
        for (int j = 0; j < 8; ++j)
            if (lane + 32 * j < dim) v[j] *= inv * w[lane + 32 * j];
    }
    template <typename T> __device__ __forceinline__ void store(T* p, uint32_t dim, uint32_t lane) const {     // zero up to pad8(dim)
#pragma unroll
        for (int j = 0; j < 8; ++j)
            if (lane + 32 * j < pad8(dim)) p[lane + 32 * j] = from_f32<T>(v[j]);
    }
};

template <typename T>
__global__ void __launch_bounds__(256) window_append_kernel(const __grid_constant__ hf2q_window_attn a, uint32_t m, T* __restrict__ q_out) {
    pdl_trigger();
    pdl_wait();
    const uint32_t lane = threadIdx.x & 31, heads = a.heads + 2 * a.kv_heads;
    const uint64_t wid = static_cast<uint64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
    if (wid >= static_cast<uint64_t>(m) * heads) return;
    const uint32_t t = static_cast<uint32_t>(wid / heads), h = static_cast<uint32_t>(wid % heads);
    const float* row = a.qkv + static_cast<size_t>(t) * a.ld;
    const uint32_t dp = pad8(a.dim), dvp = pad8(a.vdim), slot = (*a.pos + t) % a.capacity;
    HeadVec v;
    if (h < a.heads) {
        v.load(row + a.q_off + h * a.dim, a.dim, lane);
        if (a.q_norm) v.norm(a.q_norm, a.eps, a.dim, lane);
        v.store(q_out + (static_cast<size_t>(t) * a.heads + h) * dp, a.dim, lane);
    } else if (h < a.heads + a.kv_heads) {
        const uint32_t g = h - a.heads;
        v.load(row + a.k_off + g * a.dim, a.dim, lane);
        if (a.k_norm) v.norm(a.k_norm, a.eps, a.dim, lane);
        v.store(static_cast<T*>(a.k_cache) + (static_cast<size_t>(g) * a.capacity + slot) * dp, a.dim, lane);
    } else {
        const uint32_t g = h - a.heads - a.kv_heads;
        v.load(row + a.v_off + g * a.vdim, a.vdim, lane);
        v.store(static_cast<T*>(a.v_cache) + (static_cast<size_t>(g) * a.capacity + slot) * dvp, a.vdim, lane);
    }
}

// Online softmax of one warp for GR query heads against keys [lo, hi) of KV head g; qs: [GR][dp] f32 in shared
// memory, ps: [GR][32] of this warp.  Lane = key for the scores, lane = value columns 2 lane + 64 c for the sums.
template <typename T, int GR, int NC, bool PLAIN>
struct WarpAttn {
    float mx[GR], l[GR], acc[GR][NC][2];
    __device__ __forceinline__ void init() {
#pragma unroll
        for (int g = 0; g < GR; ++g) {
            mx[g] = -CUDART_INF_F;
            l[g] = 0.f;
#pragma unroll
            for (int c = 0; c < NC; ++c) acc[g][c][0] = acc[g][c][1] = 0.f;
        }
    }
    __device__ __forceinline__ void keys(const hf2q_window_attn& a, const T* kc, const T* vc, const KeyRows<T, PLAIN>* kv, const float* qs, float* ps, const float (&r1)[GR],
                                         const float (&r2)[GR], uint32_t pos, uint32_t p0, uint32_t hi) {
        const uint32_t lane = threadIdx.x & 31, dp = pad8(a.dim), dvp = pad8(a.vdim);
        uint32_t dq = dp;
        if constexpr (PLAIN) dq += kv->sp;
        const uint32_t p = p0 + lane;
        const bool live = p < hi;
        float s[GR];
#pragma unroll
        for (int g = 0; g < GR; ++g) s[g] = 0.f;
        if (live) {
            const T* kr;
            if constexpr (PLAIN) kr = kv->key(p);
            else kr = kc + static_cast<size_t>(p % a.capacity) * dp;
#pragma unroll 4
            for (uint32_t c = 0; c < dp; c += 8) {
                float k[8];
                load8(kr + c, k);
#pragma unroll
                for (int g = 0; g < GR; ++g) {
                    const float4 x = *reinterpret_cast<const float4*>(qs + g * dq + c), y = *reinterpret_cast<const float4*>(qs + g * dq + c + 4);
                    s[g] += k[0] * x.x + k[1] * x.y + k[2] * x.z + k[3] * x.w + k[4] * y.x + k[5] * y.y + k[6] * y.z + k[7] * y.w;
                }
            }
            if constexpr (PLAIN) {
                kr = kv->shared_key(p) - dp;
#pragma unroll 4
                for (uint32_t c = dp; c < dq; c += 8) {
                    float k[8];
                    load8(kr + c, k);
#pragma unroll
                    for (int g = 0; g < GR; ++g) {
                        const float4 x = *reinterpret_cast<const float4*>(qs + g * dq + c), y = *reinterpret_cast<const float4*>(qs + g * dq + c + 4);
                        s[g] += k[0] * x.x + k[1] * x.y + k[2] * x.z + k[3] * x.w + k[4] * y.x + k[5] * y.y + k[6] * y.z + k[7] * y.w;
                    }
                }
            }
        }
#pragma unroll
        for (int g = 0; g < GR; ++g) {
            const float sc = live ? score_of(s[g], a.scale, r1[g], r2[g], pos - p, a.r1 != nullptr) : -CUDART_INF_F;
            float bm = sc;
            for (int o = 16; o > 0; o >>= 1) bm = fmaxf(bm, __shfl_xor_sync(0xffffffffu, bm, o));
            const float nm = fmaxf(mx[g], bm);
            const float corr = expf(mx[g] - nm), pr = live ? expf(sc - nm) : 0.f;
            l[g] = l[g] * corr + warp_sum(pr);
            mx[g] = nm;
#pragma unroll
            for (int c = 0; c < NC; ++c) { acc[g][c][0] *= corr; acc[g][c][1] *= corr; }
            ps[g * 32 + lane] = pr;
        }
        __syncwarp();
        const uint32_t cnt = min(32u, hi - p0);
#pragma unroll 4
        for (uint32_t i = 0; i < cnt; ++i) {
            const T* vr;
            if constexpr (PLAIN) vr = kv->value(p0 + i);
            else vr = vc + static_cast<size_t>((p0 + i) % a.capacity) * dvp;
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const uint32_t d = 2 * lane + 64 * c;
                if (d < dvp) {
                    const float v0 = to_f32(vr[d]), v1 = to_f32(vr[d + 1]);
#pragma unroll
                    for (int g = 0; g < GR; ++g) {
                        const float w = ps[g * 32 + i];
                        acc[g][c][0] = fmaf(w, v0, acc[g][c][0]);
                        acc[g][c][1] = fmaf(w, v1, acc[g][c][1]);
                    }
                }
            }
        }
        __syncwarp();
    }
};

// ---------------------------------------------------------------- decode
constexpr int WD_WARPS = 8;
__host__ __device__ constexpr uint32_t wd_part(uint32_t vdim) { return 4 + pad8(vdim); }

// grid (kv_heads * groups of GR query heads, splits); scratch: counters [grid.x] (256-byte multiple), then
// [grid.x][splits][GR][max, sum, 2 pad, acc]
template <typename T, int GR, int NC>
__global__ void __launch_bounds__(WD_WARPS * 32) window_decode_kernel(const __grid_constant__ hf2q_window_attn a, uint32_t groups, float* __restrict__ out,
                                                                      uint32_t* __restrict__ counters, float* __restrict__ part) {
    extern __shared__ __align__(16) float sm[];
    const uint32_t dp = pad8(a.dim), dvp = pad8(a.vdim), PP = wd_part(a.vdim);
    float* qs = sm;                                        // [GR][dp]
    float* ps = qs + GR * dp;                              // [warps][GR][32]
    float* rm = ps + WD_WARPS * GR * 32;                   // [warps][GR] max, then sums
    float* rl = rm + WD_WARPS * GR;
    float* ra = rl + WD_WARPS * GR;                        // [warps][GR][dvp]
    __shared__ uint32_t is_last;
    pdl_trigger();
    pdl_wait();
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t kvh = blockIdx.x / groups, rep = a.heads / a.kv_heads, g0 = (blockIdx.x % groups) * GR, n_g = min(static_cast<uint32_t>(GR), rep - g0);
    const uint32_t h0 = kvh * rep + g0, split = blockIdx.y, nsplit = gridDim.y;
    const uint32_t pos = *a.pos, n = min(pos + 1, a.window), first = pos + 1 - n;
    const uint32_t chunk = (n + nsplit - 1) / nsplit;
    const uint32_t lo = first + min(split * chunk, n), hi = first + min(split * chunk + chunk, n);
    T* kc = static_cast<T*>(a.k_cache) + static_cast<size_t>(kvh) * a.capacity * dp;
    T* vc = static_cast<T*>(a.v_cache) + static_cast<size_t>(kvh) * a.capacity * dvp;
    for (uint32_t g = warp; g < GR; g += WD_WARPS) {
        HeadVec v;
        v.load(a.qkv + a.q_off + (h0 + min(g, n_g - 1)) * a.dim, a.dim, lane);
        if (a.q_norm) v.norm(a.q_norm, a.eps, a.dim, lane);
#pragma unroll
        for (int j = 0; j < 8; ++j)
            if (lane + 32 * j < dp) qs[g * dp + lane + 32 * j] = to_f32(from_f32<T>(v.v[j]));      // the prefill's operand precision
    }
    if (pos >= lo && pos < hi && warp < 2) {               // the new position, by the CTAs whose range holds it
        const uint32_t slot = pos % a.capacity;
        HeadVec v;
        if (warp == 0) {
            v.load(a.qkv + a.k_off + kvh * a.dim, a.dim, lane);
            if (a.k_norm) v.norm(a.k_norm, a.eps, a.dim, lane);
            v.store(kc + static_cast<size_t>(slot) * dp, a.dim, lane);
        } else {
            v.load(a.qkv + a.v_off + kvh * a.vdim, a.vdim, lane);
            v.store(vc + static_cast<size_t>(slot) * dvp, a.vdim, lane);
        }
    }
    float r1[GR], r2[GR];
#pragma unroll
    for (int g = 0; g < GR; ++g) {
        r1[g] = a.r1 ? a.r1[h0 + min(static_cast<uint32_t>(g), n_g - 1)] : 0.f;
        r2[g] = a.r1 ? a.r2[h0 + min(static_cast<uint32_t>(g), n_g - 1)] : 0.f;
    }
    __syncthreads();
    WarpAttn<T, GR, NC, false> w;
    w.init();
    for (uint32_t p0 = lo + warp * 32; p0 < hi; p0 += WD_WARPS * 32) w.keys(a, kc, vc, nullptr, qs, ps + warp * GR * 32, r1, r2, pos, p0, hi);
#pragma unroll
    for (int g = 0; g < GR; ++g) {
        if (lane == 0) { rm[warp * GR + g] = w.mx[g]; rl[warp * GR + g] = w.l[g]; }
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            const uint32_t d = 2 * lane + 64 * c;
            if (d < dvp) *reinterpret_cast<float2*>(ra + (warp * GR + g) * dvp + d) = make_float2(w.acc[g][c][0], w.acc[g][c][1]);
        }
    }
    __syncthreads();
    float* mine = part + (static_cast<size_t>(blockIdx.x) * nsplit + split) * GR * PP;
    for (uint32_t i = threadIdx.x; i < GR * dvp; i += WD_WARPS * 32) {
        const uint32_t g = i / dvp, d = i % dvp;
        float m = -CUDART_INF_F, l = 0.f, s = 0.f;
        for (int k = 0; k < WD_WARPS; ++k) m = fmaxf(m, rm[k * GR + g]);
        for (int k = 0; k < WD_WARPS; ++k) {
            const float c = rm[k * GR + g] == -CUDART_INF_F ? 0.f : expf(rm[k * GR + g] - m);
            l += rl[k * GR + g] * c;
            s += ra[(k * GR + g) * dvp + d] * c;
        }
        if (nsplit == 1) {
            if (g < n_g && d < a.vdim) out[(h0 + g) * a.vdim + d] = s / l;
        } else {
            if (d == 0) { mine[g * PP] = m; mine[g * PP + 1] = l; }
            mine[g * PP + 4 + d] = s;
        }
    }
    if (nsplit == 1) return;
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) {
        const uint32_t old = atomicAdd(&counters[blockIdx.x], 1u);
        is_last = old == nsplit - 1;
        if (is_last) counters[blockIdx.x] = 0;
    }
    __syncthreads();
    if (!is_last) return;
    __threadfence();
    const float* all = part + static_cast<size_t>(blockIdx.x) * nsplit * GR * PP;
    for (uint32_t i = threadIdx.x; i < n_g * a.vdim; i += WD_WARPS * 32) {
        const uint32_t g = i / a.vdim, d = i % a.vdim;
        float m = -CUDART_INF_F, l = 0.f, s = 0.f;
        for (uint32_t k = 0; k < nsplit; ++k) m = fmaxf(m, __ldcg(all + (k * GR + g) * PP));
        for (uint32_t k = 0; k < nsplit; ++k) {
            const float* src = all + (k * GR + g) * PP;
            const float mk = __ldcg(src), c = mk == -CUDART_INF_F ? 0.f : expf(mk - m);
            l += __ldcg(src + 1) * c;
            s += __ldcg(src + 4 + d) * c;
        }
        out[(h0 + g) * a.vdim + d] = s / l;
    }
}

constexpr uint32_t QK_MAX = 320;                        // dim and shared_dim together, padded

// ---------------------------------------------------------------- prefill, f32: one warp per (query, head)
template <typename T, typename OUT, int NC, bool PLAIN>
__global__ void __launch_bounds__(256) window_prefill_f32_kernel(const __grid_constant__ hf2q_window_attn a, uint32_t m, const T* __restrict__ q,
                                                                 const float* __restrict__ gate, uint32_t ldg, OUT* __restrict__ out, uint32_t ldo) {
    __shared__ __align__(16) float qs[8][QK_MAX];
    __shared__ float ps[8][32];
    pdl_trigger();
    pdl_wait();
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.y, t = blockIdx.x * 8 + warp;
    if (t >= m) return;
    const KeyRows<T, PLAIN> kv(a, h / (a.heads / a.kv_heads), *a.pos);
    const uint32_t dq = kv.dp + kv.sp;
    for (uint32_t i = lane; i < dq; i += 32) qs[warp][i] = to_f32(q[(static_cast<size_t>(t) * a.heads + h) * dq + i]);
    __syncwarp();
    const uint32_t pos = *a.pos + t, n = min(pos + 1, a.window), hi = pos + 1;
    const float r1[1] = {a.r1 ? a.r1[h] : 0.f}, r2[1] = {a.r1 ? a.r2[h] : 0.f};
    WarpAttn<T, 1, NC, PLAIN> w;
    w.init();
    for (uint32_t p0 = hi - n; p0 < hi; p0 += 32) w.keys(a, kv.k, kv.v, &kv, qs[warp], ps[warp], r1, r2, pos, p0, hi);
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const uint32_t d = 2 * lane + 64 * c + u;
            if (d < a.vdim) {
                float v = w.acc[0][c][u] / w.l[0];
                if (gate) v *= sigmoidf(gate[static_cast<size_t>(t) * ldg + h * a.vdim + d]);
                out[static_cast<size_t>(t) * ldo + h * a.vdim + d] = from_f32<OUT>(v);
            }
        }
    if (h == a.heads - 1)
        for (uint32_t i = a.heads * a.vdim + lane; i < ldo; i += 32) out[static_cast<size_t>(t) * ldo + i] = from_f32<OUT>(0.f);
}

// ---------------------------------------------------------------- prefill, bf16 cache, tensor cores
constexpr int WP_WARPS = 4, WP_Q = 16 * WP_WARPS, WP_K = 64;

// grid (query tiles, heads); DK >= dim + shared_dim, DV >= vdim.  Keys are walked from the first one the tile's first
// query sees.
template <int DK, int DV, typename OUT, bool PLAIN>
__global__ void __launch_bounds__(WP_WARPS * 32) window_prefill_mma_kernel(const __grid_constant__ hf2q_window_attn a, uint32_t m,
                                                                           const __nv_bfloat16* __restrict__ q, const float* __restrict__ gate, uint32_t ldg,
                                                                           OUT* __restrict__ out, uint32_t ldo) {
    constexpr uint32_t KP = DK + 8, VP = DV + 8, K_TILE = WP_K * KP, TILES = K_TILE + WP_K * VP;      // pitches and sizes in elements
    extern __shared__ __align__(16) __nv_bfloat16 kv[];             // [2][K tile, V tile]
    pdl_trigger();
    pdl_wait();
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, t4 = lane & 3;
    const uint32_t h = blockIdx.y, t0 = blockIdx.x * WP_Q;
    const uint32_t pos0 = *a.pos;
    const KeyRows<__nv_bfloat16, PLAIN> rows(a, h / (a.heads / a.kv_heads), pos0);
    const uint32_t dq = rows.dp + rows.sp, dvp = pad8(a.vdim), nk = (dq + 15) / 16, nv = (dvp + 15) / 16;
    const uint32_t q_lo = pos0 + t0, q_hi = pos0 + min(t0 + WP_Q, m) - 1;
    const uint32_t j0 = q_lo + 1 > a.window ? q_lo + 1 - a.window : 0u;
    // elements past dim / vdim, and keys never loaded, must be finite zeros
    for (uint32_t i = threadIdx.x; i < 2 * TILES / 8; i += WP_WARPS * 32) reinterpret_cast<uint4*>(kv)[i] = make_uint4(0, 0, 0, 0);
    __syncthreads();
    auto stage = [&](uint32_t key0, uint32_t b) {
        __nv_bfloat16* ks = kv + b * TILES;
        __nv_bfloat16* vs = ks + K_TILE;
        const uint32_t ck = dq / 8, cv = dvp / 8, cd = rows.dp / 8;
        for (uint32_t i = threadIdx.x; i < WP_K * ck; i += WP_WARPS * 32) {
            const uint32_t r = i / ck, c = i % ck;
            if (key0 + r <= q_hi) cp_async16(ks + r * KP + 8 * c, !PLAIN || c < cd ? rows.key(key0 + r) + 8 * c : rows.shared_key(key0 + r) + 8 * (c - cd));
        }
        for (uint32_t i = threadIdx.x; i < WP_K * cv; i += WP_WARPS * 32) {
            const uint32_t r = i / cv, c = i % cv;
            if (key0 + r <= q_hi) cp_async16(vs + r * VP + 8 * c, rows.value(key0 + r) + 8 * c);
        }
        cp_async_commit();
    };
    stage(j0, 0);
    uint32_t qa[DK / 16][4];
    uint32_t row[2], qpos[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) { row[u] = t0 + warp * 16 + gid + 8 * u; qpos[u] = pos0 + row[u]; }
#pragma unroll
    for (int k = 0; k < DK / 16; ++k)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const uint32_t r = row[i & 1], c = 16 * k + 8 * (i >> 1) + 2 * t4;
            qa[k][i] = r < m && c < dq ? *reinterpret_cast<const uint32_t*>(q + (static_cast<size_t>(r) * a.heads + h) * dq + c) : 0u;
        }
    const bool bias = a.r1 != nullptr;
    const float r1 = bias ? a.r1[h] : 0.f, r2 = bias ? a.r2[h] : 0.f;
    float mx[2] = {-CUDART_INF_F, -CUDART_INF_F}, l[2] = {0.f, 0.f};
    float o[DV / 8][4];
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    const uint32_t n_tiles = (q_hi - j0) / WP_K + 1;
    const uint32_t w_lo = pos0 + t0 + warp * 16, w_hi = w_lo + 15;           // this warp's query positions
    for (uint32_t kt = 0; kt < n_tiles; ++kt) {
        const uint32_t key0 = j0 + kt * WP_K, b = kt & 1;
        if (kt + 1 < n_tiles) { stage(key0 + WP_K, b ^ 1); cp_async_wait<1>(); }
        else cp_async_wait<0>();
        __syncthreads();
        // keys above this warp's last query or below its first window edge touch none of its rows
        if (key0 <= w_hi && key0 + WP_K - 1 + a.window > w_lo) {
            const uint32_t ks = smem_u32(kv + b * TILES), vs = ks + K_TILE * 2;
            float s[WP_K / 8][4];
#pragma unroll
            for (int i = 0; i < WP_K / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
#pragma unroll
            for (int k = 0; k < DK / 16; ++k) {
                if (k < static_cast<int>(nk)) {
#pragma unroll
                    for (int n2 = 0; n2 < WP_K / 16; ++n2) {
                        uint32_t f[4];
                        ldmatrix4(f, ks + ((n2 * 16 + (lane >> 4) * 8 + (lane & 7)) * KP + 16 * k + ((lane >> 3) & 1) * 8) * 2);
                        mma_bf16(s[2 * n2], qa[k], f[0], f[1]);
                        mma_bf16(s[2 * n2 + 1], qa[k], f[2], f[3]);
                    }
                }
            }
            float bm[2] = {-CUDART_INF_F, -CUDART_INF_F};
#pragma unroll
            for (int n = 0; n < WP_K / 8; ++n)
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const uint32_t key = key0 + 8 * n + 2 * t4 + (i & 1), qp = qpos[i >> 1];
                    const uint32_t dist = qp - key;                          // wraps to a huge value for keys after the query
                    float v = s[n][i] * a.scale;
                    if (bias) v -= r1 * __logf(fmaf(r2, static_cast<float>(dist), 1.0f));
                    v = dist < a.window ? v : -CUDART_INF_F;
                    s[n][i] = v;
                    bm[i >> 1] = fmaxf(bm[i >> 1], v);
                }
            float nm[2];
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                bm[u] = fmaxf(bm[u], __shfl_xor_sync(0xffffffffu, bm[u], 1));
                bm[u] = fmaxf(bm[u], __shfl_xor_sync(0xffffffffu, bm[u], 2));
                const float top = fmaxf(mx[u], bm[u]);
                nm[u] = top == -CUDART_INF_F ? 0.f : top;                    // nothing visible yet: every weight is exp(-inf) = 0
                const float corr = __expf(mx[u] - nm[u]);
                l[u] *= corr;
                mx[u] = top;
#pragma unroll
                for (int i = 0; i < DV / 8; ++i) { o[i][2 * u] *= corr; o[i][2 * u + 1] *= corr; }
            }
#pragma unroll
            for (int n = 0; n < WP_K / 8; ++n)
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    s[n][i] = __expf(s[n][i] - nm[i >> 1]);
                    l[i >> 1] += s[n][i];                                    // this lane's share; summed over the four lanes at the end
                }
#pragma unroll
            for (int k = 0; k < WP_K / 16; ++k) {
                uint32_t pa[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) pa[i] = pack_bf16(s[2 * k + (i >> 1)][2 * (i & 1)], s[2 * k + (i >> 1)][2 * (i & 1) + 1]);
#pragma unroll
                for (int n2 = 0; n2 < DV / 16; ++n2) {
                    if (n2 < static_cast<int>(nv)) {
                        uint32_t f[4];
                        ldmatrix4_trans(f, vs + ((16 * k + ((lane >> 3) & 1) * 8 + (lane & 7)) * VP + 16 * n2 + (lane >> 4) * 8) * 2);
                        mma_bf16(o[2 * n2], pa, f[0], f[1]);
                        mma_bf16(o[2 * n2 + 1], pa, f[2], f[3]);
                    }
                }
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int u = 0; u < 2; ++u) {
        l[u] += __shfl_xor_sync(0xffffffffu, l[u], 1);
        l[u] += __shfl_xor_sync(0xffffffffu, l[u], 2);
        if (row[u] >= m) continue;
        const float inv = 1.0f / l[u];
        OUT* dst = out + static_cast<size_t>(row[u]) * ldo + h * a.vdim;
        const float* gr = gate ? gate + static_cast<size_t>(row[u]) * ldg + h * a.vdim : nullptr;
#pragma unroll
        for (int n = 0; n < DV / 8; ++n)
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const uint32_t d = 8 * n + 2 * t4 + i;
                if (d < a.vdim) {
                    float v = o[n][2 * u + i] * inv;
                    if (gr) v *= sigmoidf(gr[d]);
                    dst[d] = from_f32<OUT>(v);
                }
            }
        if (h == a.heads - 1)
            for (uint32_t i = a.heads * a.vdim + t4; i < ldo; i += 4) out[static_cast<size_t>(row[u]) * ldo + i] = from_f32<OUT>(0.f);
    }
}

// ---------------------------------------------------------------- host side
bool window_ok(const hf2q_window_attn* a) {
    return a && a->qkv && a->k_cache && a->v_cache && a->pos && a->heads && a->kv_heads && a->heads % a->kv_heads == 0 && a->dim && a->dim <= 256 &&
           a->vdim && a->vdim <= 256 && a->window && a->capacity >= a->window && (a->r1 == nullptr) == (a->r2 == nullptr) &&
           (a->cache_dtype == HF2Q_DT_F32 || a->cache_dtype == HF2Q_DT_BF16) && reinterpret_cast<uintptr_t>(a->k_cache) % 16 == 0 &&
           reinterpret_cast<uintptr_t>(a->v_cache) % 16 == 0 && !a->linear && !a->shared_dim;
}
// what the prefill takes beyond that: plain rows, a shared part of the keys
bool window_rows_ok(const hf2q_window_attn* a) {
    if (!a || !a->linear) return window_ok(a);
    hf2q_window_attn b = *a;
    b.qkv = b.qkv ? b.qkv : static_cast<const float*>(a->k_cache);           // the queries come apart
    b.linear = b.shared_dim = 0;
    const bool shared = a->shared_dim == 0 || (a->k_shared && a->shared_capacity && a->shared_stride % 8 == 0 && a->shared_stride >= pad8(a->shared_dim) &&
                                               reinterpret_cast<uintptr_t>(a->k_shared) % 16 == 0 && pad8(a->dim) + pad8(a->shared_dim) <= QK_MAX);
    return window_ok(&b) && shared && (!a->linear || (a->row_stride % 8 == 0 && a->k_head_stride % 8 == 0 && a->v_head_stride % 8 == 0));
}
uint32_t decode_gr(const hf2q_window_attn& a) {
    const uint32_t rep = a.heads / a.kv_heads;
    return rep >= 5 ? 8 : rep >= 3 ? 4 : rep;
}
uint32_t decode_groups(const hf2q_window_attn& a) { const uint32_t gr = decode_gr(a); return (a.heads / a.kv_heads + gr - 1) / gr; }
uint32_t decode_splits(const hf2q_window_attn& a, int sms) {
    const uint32_t ctas = a.kv_heads * decode_groups(a), by_sm = (2 * sms + ctas - 1) / ctas, by_keys = (a.window + 127) / 128;
    const uint32_t s = by_sm < by_keys ? by_sm : by_keys;
    return s < 1 ? 1 : s > 64 ? 64 : s;
}
size_t counter_bytes(const hf2q_window_attn& a) { return (static_cast<size_t>(a.kv_heads) * decode_groups(a) * 4 + 255) & ~static_cast<size_t>(255); }

template <typename T, int GR, int NC>
cudaError_t launch_decode(const hf2q_window_attn& a, float* out, uint8_t* scratch, int sms, cudaStream_t st) {
    static PerDeviceFlag flag;
    const size_t smem = (static_cast<size_t>(GR) * pad8(a.dim) + WD_WARPS * GR * (34 + pad8(a.vdim))) * sizeof(float);
    if (const cudaError_t e = ensure_max_dynamic_smem(window_decode_kernel<T, GR, NC>, 100 * 1024, flag); e != cudaSuccess) return e;
    const uint32_t groups = decode_groups(a);
    return launch_pdl(window_decode_kernel<T, GR, NC>, dim3(a.kv_heads * groups, decode_splits(a, sms)), dim3(WD_WARPS * 32), smem, st, a, groups, out,
                      reinterpret_cast<uint32_t*>(scratch), reinterpret_cast<float*>(scratch + counter_bytes(a)));
}
template <typename T, int GR>
cudaError_t launch_decode_nc(const hf2q_window_attn& a, float* out, uint8_t* scratch, int sms, cudaStream_t st) {
    if (a.vdim <= 64) return launch_decode<T, GR, 1>(a, out, scratch, sms, st);
    if (a.vdim <= 128) return launch_decode<T, GR, 2>(a, out, scratch, sms, st);
    return launch_decode<T, GR, 4>(a, out, scratch, sms, st);
}
template <typename T>
cudaError_t launch_decode_gr(const hf2q_window_attn& a, float* out, uint8_t* scratch, int sms, cudaStream_t st) {
    switch (decode_gr(a)) {
        case 1: return launch_decode_nc<T, 1>(a, out, scratch, sms, st);
        case 2: return launch_decode_nc<T, 2>(a, out, scratch, sms, st);
        case 4: return launch_decode_nc<T, 4>(a, out, scratch, sms, st);
        default: return launch_decode_nc<T, 8>(a, out, scratch, sms, st);
    }
}
template <typename T, typename OUT, bool PLAIN>
cudaError_t launch_prefill_f32(const hf2q_window_attn& a, uint32_t m, const void* q, const float* gate, uint32_t ldg, void* out, uint32_t ldo, cudaStream_t st) {
    const dim3 grid((m + 7) / 8, a.heads);
    const T* qt = static_cast<const T*>(q);
    OUT* o = static_cast<OUT*>(out);
    if (a.vdim <= 64) return launch_pdl(window_prefill_f32_kernel<T, OUT, 1, PLAIN>, grid, dim3(256), 0, st, a, m, qt, gate, ldg, o, ldo);
    if (a.vdim <= 128) return launch_pdl(window_prefill_f32_kernel<T, OUT, 2, PLAIN>, grid, dim3(256), 0, st, a, m, qt, gate, ldg, o, ldo);
    return launch_pdl(window_prefill_f32_kernel<T, OUT, 4, PLAIN>, grid, dim3(256), 0, st, a, m, qt, gate, ldg, o, ldo);
}
template <int DK, int DV, typename OUT, bool PLAIN>
cudaError_t launch_prefill_dm(const hf2q_window_attn& a, uint32_t m, const void* q, const float* gate, uint32_t ldg, void* out, uint32_t ldo, cudaStream_t st) {
    static PerDeviceFlag flag;
    const size_t smem = 2ull * WP_K * (DK + 8 + DV + 8) * 2;
    if (const cudaError_t e = ensure_max_dynamic_smem(window_prefill_mma_kernel<DK, DV, OUT, PLAIN>, static_cast<int>(smem), flag); e != cudaSuccess) return e;
    return launch_pdl(window_prefill_mma_kernel<DK, DV, OUT, PLAIN>, dim3((m + WP_Q - 1) / WP_Q, a.heads), dim3(WP_WARPS * 32), smem, st, a, m,
                      static_cast<const __nv_bfloat16*>(q), gate, ldg, static_cast<OUT*>(out), ldo);
}
template <typename OUT>
cudaError_t launch_prefill_mma(const hf2q_window_attn& a, uint32_t m, const void* q, const float* gate, uint32_t ldg, void* out, uint32_t ldo, cudaStream_t st) {
    const uint32_t k = pad8(a.dim) + pad8(a.shared_dim), v = a.vdim;
    if (a.linear) {
        if (k <= 64 && v <= 64) return launch_prefill_dm<64, 64, OUT, true>(a, m, q, gate, ldg, out, ldo, st);
        if (k <= 128 && v <= 128) return launch_prefill_dm<128, 128, OUT, true>(a, m, q, gate, ldg, out, ldo, st);
        if (k <= 192 && v <= 128) return launch_prefill_dm<192, 128, OUT, true>(a, m, q, gate, ldg, out, ldo, st);
        return launch_prefill_dm<QK_MAX, 256, OUT, true>(a, m, q, gate, ldg, out, ldo, st);
    }
    if (k <= 64 && v <= 64) return launch_prefill_dm<64, 64, OUT, false>(a, m, q, gate, ldg, out, ldo, st);
    if (k <= 128 && v <= 128) return launch_prefill_dm<128, 128, OUT, false>(a, m, q, gate, ldg, out, ldo, st);
    return launch_prefill_dm<256, 256, OUT, false>(a, m, q, gate, ldg, out, ldo, st);
}

}  // namespace
}  // namespace hf2q

using namespace hf2q;
using namespace hf2q::seq;

extern "C" {

HF2Q_API int32_t hf2q_cuda_window_attn_scratch_bytes(hf2q_ctx* ctx, const hf2q_window_attn* a, uint64_t* out) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!a || !out || a->kv_heads == 0 || a->heads == 0 || a->heads % a->kv_heads || a->window == 0)
        return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "window_attn_scratch_bytes: bad sizes");
    *out = counter_bytes(*a) + static_cast<uint64_t>(a->kv_heads) * decode_groups(*a) * decode_splits(*a, ctx_sm_count(ctx)) * decode_gr(*a) * wd_part(a->vdim) * 4;
    return HF2Q_OK;
}

HF2Q_API int32_t hf2q_cuda_window_attn_decode(hf2q_ctx* ctx, void* stream, const hf2q_window_attn* a, float* out, void* scratch, uint64_t scratch_bytes) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    uint64_t need = 0;
    if (!window_ok(a) || !out || !scratch || hf2q_cuda_window_attn_scratch_bytes(ctx, a, &need) != HF2Q_OK)
        return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "window_attn_decode: null pointer or an unsupported size");
    if (scratch_bytes < need) return ctx_fail(ctx, HF2Q_ERR_WORKSPACE, "window_attn_decode: scratch too small");
    const cudaStream_t st = static_cast<cudaStream_t>(stream);
    const int sms = ctx_sm_count(ctx);
    const cudaError_t e = a->cache_dtype == HF2Q_DT_F32 ? launch_decode_gr<float>(*a, out, static_cast<uint8_t*>(scratch), sms, st)
                                                        : launch_decode_gr<__nv_bfloat16>(*a, out, static_cast<uint8_t*>(scratch), sms, st);
    return ctx_cuda_result(ctx, e, "window_attn_decode", 1);
}

HF2Q_API int32_t hf2q_cuda_window_attn_append(hf2q_ctx* ctx, void* stream, const hf2q_window_attn* a, uint32_t m, void* q_out) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!window_ok(a) || !q_out || a->window - 1 + static_cast<uint64_t>(m) > a->capacity)
        return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "window_attn_append: null pointer, an unsupported size or more tokens than the ring holds");
    if (m == 0) return HF2Q_OK;
    const uint64_t warps = static_cast<uint64_t>(m) * (a->heads + 2 * a->kv_heads);
    const dim3 grid(static_cast<unsigned>((warps + 7) / 8));
    const cudaStream_t st = static_cast<cudaStream_t>(stream);
    const cudaError_t e = a->cache_dtype == HF2Q_DT_F32 ? launch_pdl(window_append_kernel<float>, grid, dim3(256), 0, st, *a, m, static_cast<float*>(q_out))
                                                        : launch_pdl(window_append_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, *a, m, static_cast<__nv_bfloat16*>(q_out));
    return ctx_cuda_result(ctx, e, "window_attn_append", 1);
}

HF2Q_API int32_t hf2q_cuda_window_attn_prefill(hf2q_ctx* ctx, void* stream, const hf2q_window_attn* a, uint32_t m, const void* q, const float* gate,
                                               uint32_t ldg, void* out, uint32_t out_dtype, uint32_t ldo) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!window_rows_ok(a) || !q || !out || ldo < a->heads * a->vdim || a->window - 1 + static_cast<uint64_t>(m) > a->capacity)
        return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "window_attn_prefill: null pointer, an unsupported size or more tokens than the ring holds");
    if (m == 0) return HF2Q_OK;
    const cudaStream_t st = static_cast<cudaStream_t>(stream);
    cudaError_t e = cudaErrorInvalidValue;
    if (a->cache_dtype == HF2Q_DT_F32) {
        if (out_dtype == HF2Q_DT_F32)
            e = a->linear ? launch_prefill_f32<float, float, true>(*a, m, q, gate, ldg, out, ldo, st) : launch_prefill_f32<float, float, false>(*a, m, q, gate, ldg, out, ldo, st);
    } else if (out_dtype == HF2Q_DT_BF16) {
        e = launch_prefill_mma<__nv_bfloat16>(*a, m, q, gate, ldg, out, ldo, st);
    } else if (out_dtype == HF2Q_DT_F32) {
        e = launch_prefill_mma<float>(*a, m, q, gate, ldg, out, ldo, st);
    }
    return ctx_cuda_result(ctx, e, "window_attn_prefill", 1);
}

}  // extern "C"
