// Latent attention over a sliding window: the cache holds one normed latent vector and one rotated key part per token
// (ring, position p in slot p % capacity), shared by all heads.
//
//   append   prefill: latents and rotated key parts to the cache, rotated queries to a buffer; the caller expands the
//            window's latents to keys and values with a product and runs the windowed prefill over them
//   decode   three launches: the query moves into the latent space (q . uk c = (uk^T q) . c), attention over the cached
//            rows with all heads sharing a tile of them (bf16: on the tensor cores; f32: in f32), then the merge of the
//            splits and the heads' value matrices
#include <cooperative_groups.h>
#include <math_constants.h>

#include "mma_sync.cuh"
#include "seq_common.cuh"

namespace hf2q {
namespace {
using namespace seq;

__host__ __device__ constexpr uint32_t pad8(uint32_t n) { return (n + 7) & ~7u; }
__host__ __device__ inline uint32_t row_elems(const hf2q_latent_attn& a) { return pad8(a.kv_rank) + pad8(a.rot_dim); }

// element i of a vector whose first `pairs` pairs (2i, 2i + 1) turn by pos * freq
__device__ __forceinline__ float rotated(const float* v, uint32_t i, uint32_t pairs, const float* freq, uint32_t pos) {
    if (i >= 2 * pairs) return v[i];
    float s, c;
    sincosf(static_cast<float>(pos) * freq[i / 2], &s, &c);
    const float u = v[i & ~1u], w = v[i | 1u];
    return i & 1 ? w * c + u * s : u * c - w * s;
}

// the cache row of one token, by one warp
template <typename T>
__device__ __forceinline__ void append_row(const hf2q_latent_attn& a, const float* src, uint32_t pos) {
    const uint32_t lane = threadIdx.x & 31, rp = pad8(a.kv_rank), sp = pad8(a.rot_dim);
    T* dst = static_cast<T*>(a.cache) + static_cast<size_t>(pos % a.capacity) * (rp + sp);
    float s = 0.f;
    for (uint32_t i = lane; i < a.kv_rank; i += 32) s += src[i] * src[i];
    const float inv = 1.0f / sqrtf(warp_sum(s) / static_cast<float>(a.kv_rank) + a.eps);
    for (uint32_t i = lane; i < rp; i += 32) dst[i] = from_f32<T>(i < a.kv_rank ? src[i] * inv * a.norm[i] : 0.f);
    for (uint32_t i = lane; i < sp; i += 32) dst[rp + i] = from_f32<T>(i < a.rot_dim ? rotated(src + a.kv_rank, i, a.rot_pairs, a.freq, pos) : 0.f);
}

template <typename T>
__global__ void __launch_bounds__(256) latent_append_kernel(const __grid_constant__ hf2q_latent_attn a, uint32_t m, T* __restrict__ q_out) {
    pdl_trigger();
    pdl_wait();
    const uint32_t lane = threadIdx.x & 31;
    const uint64_t wid = static_cast<uint64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
    if (wid >= static_cast<uint64_t>(m) * (a.heads + 1)) return;
    const uint32_t t = static_cast<uint32_t>(wid / (a.heads + 1)), h = static_cast<uint32_t>(wid % (a.heads + 1)), pos = *a.pos + t;
    const float* row = a.proj + static_cast<size_t>(t) * a.ld;
    if (h == a.heads) {
        append_row<T>(a, row + a.c_off, pos);
        return;
    }
    const uint32_t dp = pad8(a.dim), sp = pad8(a.rot_dim);
    const float* q = row + a.q_off + h * (a.dim + a.rot_dim);
    T* dst = q_out + (static_cast<size_t>(t) * a.heads + h) * (dp + sp);
    for (uint32_t i = lane; i < dp; i += 32) dst[i] = from_f32<T>(i < a.dim ? q[i] : 0.f);
    for (uint32_t i = lane; i < sp; i += 32) dst[dp + i] = from_f32<T>(i < a.rot_dim ? rotated(q + a.dim, i, a.rot_pairs, a.freq, pos) : 0.f);
}

// ---------------------------------------------------------------- decode
// grid heads * slices + 1: a CTA takes LQ_ROWS rows of a head's uk^T; the last one appends the token.
// qa [heads][row]: latent query, rotated part; zeros in the padding
constexpr uint32_t LQ_ROWS = 128, LD_DIM = 512;

template <typename T>
__global__ void __launch_bounds__(256) latent_query_kernel(const __grid_constant__ hf2q_latent_attn a, uint32_t slices, float* __restrict__ qa) {
    __shared__ __align__(16) float q[LD_DIM];
    pdl_trigger();
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (blockIdx.x < a.heads * slices) {                                    // weights: towards L2 before the wait
        const uint32_t r0 = blockIdx.x % slices * LQ_ROWS, rows = min(LQ_ROWS, a.kv_rank - min(r0, a.kv_rank)), line = pad8(a.dim) * 2;
        const char* w = static_cast<const char*>(a.uk_t) + (static_cast<size_t>(blockIdx.x / slices) * a.kv_rank + r0) * line;
        for (uint32_t i = 128 * threadIdx.x; i < rows * line; i += 128 * 256) prefetch_l2(w + i);
    }
    pdl_wait();
    const uint32_t pos = *a.pos;
    if (blockIdx.x == a.heads * slices) {
        if (warp == 0) append_row<T>(a, a.proj + a.c_off, pos);
        return;
    }
    const uint32_t h = blockIdx.x / slices, slice = blockIdx.x % slices, dp = pad8(a.dim), rp = pad8(a.kv_rank), sp = pad8(a.rot_dim);
    const float* src = a.proj + a.q_off + h * (a.dim + a.rot_dim);
    float* dst = qa + static_cast<size_t>(h) * (rp + sp);
    for (uint32_t i = threadIdx.x; i < dp; i += 256) q[i] = i < a.dim ? src[i] : 0.f;
    if (slice == 0)
        for (uint32_t i = threadIdx.x; i < sp; i += 256) dst[rp + i] = i < a.rot_dim ? rotated(src + a.dim, i, a.rot_pairs, a.freq, pos) : 0.f;
    __syncthreads();
    // lanes in groups of eight share a row
    const uint32_t r_end = min((slice + 1) * LQ_ROWS, rp);
    float s[LQ_ROWS / 32];
#pragma unroll
    for (uint32_t j = 0; j < LQ_ROWS / 32; ++j) {
        const uint32_t r = slice * LQ_ROWS + 32 * j + warp * 4 + (lane >> 3);
        s[j] = 0.f;
        if (r < a.kv_rank) {
            const __nv_bfloat16* w = static_cast<const __nv_bfloat16*>(a.uk_t) + (static_cast<size_t>(h) * a.kv_rank + r) * dp;
#pragma unroll 2
            for (uint32_t c = 8 * (lane & 7); c < dp; c += 64) {
                float f[8];
                load8(w + c, f);
#pragma unroll
                for (int i = 0; i < 8; ++i) s[j] = fmaf(f[i], q[c + i], s[j]);
            }
        }
    }
#pragma unroll
    for (uint32_t j = 0; j < LQ_ROWS / 32; ++j) {
        const uint32_t r = slice * LQ_ROWS + 32 * j + warp * 4 + (lane >> 3);
#pragma unroll
        for (int o = 4; o > 0; o >>= 1) s[j] += __shfl_xor_sync(0xffffffffu, s[j], o);
        if ((lane & 7) == 0 && r < r_end) dst[r] = s[j];
    }
}

constexpr uint32_t LD_WARPS = 8, LD_KEYS = 32;
__host__ __device__ inline uint32_t part_elems(const hf2q_latent_attn& a) { return 4 + pad8(a.kv_rank); }

// grid (groups of 8 NH heads, splits); a warp owns NH heads, a tile of 32 keys is shared by the CTA (lane = key for the
// scores, lane = latent elements 2 lane + 64 c for the sums).  part [split][head][max, sum, 2 pad, acc]
template <typename T, int NH, int NC>
__global__ void __launch_bounds__(LD_WARPS * 32) latent_decode_kernel(const __grid_constant__ hf2q_latent_attn a, uint32_t bufs,
                                                                      const float* __restrict__ qa, float* __restrict__ part) {
    extern __shared__ __align__(16) uint8_t lsm[];
    const uint32_t rp = pad8(a.kv_rank), row = row_elems(a), pitch = row + 16 / sizeof(T);
    float* qs = reinterpret_cast<float*>(lsm);                             // [8 NH][row]
    T* tile = reinterpret_cast<T*>(qs + LD_WARPS * NH * row);              // [bufs][32][pitch]
    __shared__ float ps[LD_WARPS][NH][LD_KEYS];
    pdl_trigger();
    pdl_wait();
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, split = blockIdx.y, nsplit = gridDim.y;
    const uint32_t h_cta = blockIdx.x * LD_WARPS * NH, h0 = h_cta + warp * NH;
    const uint32_t pos = *a.pos, n = min(pos + 1, a.window), first = pos + 1 - n, chunk = (n + nsplit - 1) / nsplit;
    const uint32_t lo = first + min(split * chunk, n), hi = first + min(split * chunk + chunk, n);
    const T* cache = static_cast<const T*>(a.cache);
    auto stage = [&](uint32_t p0, uint32_t b) {
        constexpr uint32_t E = 16 / sizeof(T);
        const uint32_t per = row / E, cnt = min(LD_KEYS, hi - p0);
        for (uint32_t i = threadIdx.x; i < cnt * per; i += LD_WARPS * 32)
            cp_async16(tile + (b * LD_KEYS + i / per) * pitch + (i % per) * E, cache + static_cast<size_t>((p0 + i / per) % a.capacity) * row + (i % per) * E);
        cp_async_commit();
    };
    if (lo < hi) stage(lo, 0);
    for (uint32_t i = threadIdx.x; i < LD_WARPS * NH * row; i += LD_WARPS * 32) {
        const uint32_t h = h_cta + i / row;
        qs[i] = h < a.heads ? qa[static_cast<size_t>(h) * row + i % row] : 0.f;
    }
    float mx[NH], l[NH], acc[NH][NC][2];
#pragma unroll
    for (int g = 0; g < NH; ++g) {
        mx[g] = -CUDART_INF_F;
        l[g] = 0.f;
#pragma unroll
        for (int c = 0; c < NC; ++c) acc[g][c][0] = acc[g][c][1] = 0.f;
    }
    for (uint32_t p0 = lo, b = 0; p0 < hi; p0 += LD_KEYS) {
        const bool ahead = bufs == 2 && p0 + LD_KEYS < hi;
        if (ahead) { stage(p0 + LD_KEYS, b ^ 1); cp_async_wait<1>(); }
        else cp_async_wait<0>();
        __syncthreads();
        const uint32_t cnt = min(LD_KEYS, hi - p0);
        const T* rows = tile + b * LD_KEYS * pitch;
        float s[NH];
#pragma unroll
        for (int g = 0; g < NH; ++g) s[g] = 0.f;
        if (lane < cnt) {
            const T* kr = rows + lane * pitch;
#pragma unroll 2
            for (uint32_t c = 0; c < row; c += 8) {
                float k[8];
                load8(kr + c, k);
#pragma unroll
                for (int g = 0; g < NH; ++g) {
                    const float* q = qs + (warp * NH + g) * row + c;
                    const float4 x = *reinterpret_cast<const float4*>(q), y = *reinterpret_cast<const float4*>(q + 4);
                    s[g] += k[0] * x.x + k[1] * x.y + k[2] * x.z + k[3] * x.w + k[4] * y.x + k[5] * y.y + k[6] * y.z + k[7] * y.w;
                }
            }
        }
#pragma unroll
        for (int g = 0; g < NH; ++g) {
            const float sc = lane < cnt ? s[g] * a.scale : -CUDART_INF_F;
            float bm = sc;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) bm = fmaxf(bm, __shfl_xor_sync(0xffffffffu, bm, o));
            const float nm = fmaxf(mx[g], bm), corr = expf(mx[g] - nm), pr = lane < cnt ? expf(sc - nm) : 0.f;
            l[g] = l[g] * corr + warp_sum(pr);
            mx[g] = nm;
#pragma unroll
            for (int c = 0; c < NC; ++c) { acc[g][c][0] *= corr; acc[g][c][1] *= corr; }
            ps[warp][g][lane] = pr;
        }
        __syncwarp();
#pragma unroll 2
        for (uint32_t i = 0; i < cnt; ++i) {
            const T* vr = rows + i * pitch;
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                const uint32_t d = 2 * lane + 64 * c;
                if (d < rp) {
                    const float v0 = to_f32(vr[d]), v1 = to_f32(vr[d + 1]);
#pragma unroll
                    for (int g = 0; g < NH; ++g) {
                        acc[g][c][0] = fmaf(ps[warp][g][i], v0, acc[g][c][0]);
                        acc[g][c][1] = fmaf(ps[warp][g][i], v1, acc[g][c][1]);
                    }
                }
            }
        }
        __syncthreads();
        if (bufs == 2) b ^= 1;
        else if (p0 + LD_KEYS < hi) stage(p0 + LD_KEYS, 0);
    }
#pragma unroll
    for (int g = 0; g < NH; ++g) {
        if (h0 + g >= a.heads) continue;
        float* dst = part + (static_cast<size_t>(split) * a.heads + h0 + g) * part_elems(a);
        if (lane == 0) { dst[0] = mx[g]; dst[1] = l[g]; }
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            const uint32_t d = 2 * lane + 64 * c;
            if (d < rp) *reinterpret_cast<float2*>(dst + 4 + d) = make_float2(acc[g][c][0], acc[g][c][1]);
        }
    }
}

// bf16 cache: grid (groups of 16 MT heads, splits); tiles of 64 keys.  Scores: a warp takes 8 keys of the tile for all heads;
// sums: a warp takes 8 NT latent elements for all heads.  kv_rank <= 64 NT.  The splits of a cluster merge theirs through
// distributed shared memory: part [splits / cluster][head][...].
constexpr uint32_t LT_CLUSTER = 8, LT_KEYS = 64, LT_SP = LT_KEYS + 4, LT_PP = LT_KEYS + 8;
__host__ __device__ inline uint32_t tile_pitch(const hf2q_latent_attn& a) { return ((row_elems(a) + 31) & ~31u) + 8; }

template <int MT, int NT>
__global__ void __launch_bounds__(LD_WARPS * 32) latent_decode_mma_kernel(const __grid_constant__ hf2q_latent_attn a, uint32_t bufs,
                                                                          const float* __restrict__ qa, float* __restrict__ part) {
    extern __shared__ __align__(16) uint8_t lsm[];
    constexpr uint32_t HG = 16 * MT;
    const uint32_t rp = pad8(a.kv_rank), row = row_elems(a), pitch = tile_pitch(a), ks = (pitch - 8) / 32;
    __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(lsm);             // [HG][pitch]
    __nv_bfloat16* tile = qs + HG * pitch;                                 // [bufs][64][pitch]
    float* sc = reinterpret_cast<float*>(tile + bufs * LT_KEYS * pitch);   // [HG][LT_SP]
    __nv_bfloat16* ps = reinterpret_cast<__nv_bfloat16*>(sc + HG * LT_SP); // [HG][LT_PP]
    __shared__ float corr[HG], stats[HG][2], weight[LT_CLUSTER][HG];
    pdl_trigger();
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, t4 = lane & 3, split = blockIdx.y, nsplit = gridDim.y;
    const uint32_t h_cta = blockIdx.x * HG;
    // the padding behind a row must be finite
    const uint32_t pad = (pitch - row) / 8;
    for (uint32_t i = threadIdx.x; i < bufs * LT_KEYS * pad; i += LD_WARPS * 32) *reinterpret_cast<uint4*>(tile + i / pad * pitch + row + i % pad * 8) = make_uint4(0, 0, 0, 0);
    pdl_wait();
    const uint32_t pos = *a.pos, n = min(pos + 1, a.window), first = pos + 1 - n;
    const uint32_t chunk = ((n + nsplit - 1) / nsplit + LT_KEYS - 1) / LT_KEYS * LT_KEYS;
    const uint32_t lo = first + min(split * chunk, n), hi = first + min(split * chunk + chunk, n);
    const __nv_bfloat16* cache = static_cast<const __nv_bfloat16*>(a.cache);
    auto stage = [&](uint32_t p0, uint32_t b) {
        const uint32_t per = row / 8, cnt = min(LT_KEYS, hi - p0);
        for (uint32_t i = threadIdx.x; i < cnt * per; i += LD_WARPS * 32)
            cp_async16(tile + (b * LT_KEYS + i / per) * pitch + i % per * 8, cache + static_cast<size_t>((p0 + i / per) % a.capacity) * row + i % per * 8);
        for (uint32_t i = cnt * per + threadIdx.x; i < LT_KEYS * per; i += LD_WARPS * 32)       // keys past the end: finite
            *reinterpret_cast<uint4*>(tile + (b * LT_KEYS + i / per) * pitch + i % per * 8) = make_uint4(0, 0, 0, 0);
        cp_async_commit();
    };
    if (lo < hi) stage(lo, 0);
    for (uint32_t i = threadIdx.x; i < HG * (pitch / 2); i += LD_WARPS * 32) {
        const uint32_t g = i / (pitch / 2), c = 2 * (i % (pitch / 2)), h = h_cta + g;
        const float2 v = h < a.heads && c < row ? *reinterpret_cast<const float2*>(qa + static_cast<size_t>(h) * row + c) : make_float2(0.f, 0.f);
        reinterpret_cast<uint32_t*>(qs)[i] = pack_bf16(v.x, v.y);
    }
    constexpr int HW = HG / LD_WARPS;                                      // heads whose softmax this warp keeps
    float mx[HW], l[HW], o[MT][NT][4];
#pragma unroll
    for (int g = 0; g < HW; ++g) { mx[g] = -CUDART_INF_F; l[g] = 0.f; }
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int c = 0; c < NT; ++c) o[m][c][0] = o[m][c][1] = o[m][c][2] = o[m][c][3] = 0.f;
    const uint32_t col0 = warp * 8 * NT;
    for (uint32_t p0 = lo, b = 0; p0 < hi; p0 += LT_KEYS) {
        if (bufs == 2 && p0 + LT_KEYS < hi) { stage(p0 + LT_KEYS, b ^ 1); cp_async_wait<1>(); }
        else cp_async_wait<0>();
        __syncthreads();
        const uint32_t cnt = min(LT_KEYS, hi - p0), ts = smem_u32(tile + b * LT_KEYS * pitch);
        float s[MT][4];
#pragma unroll
        for (int m = 0; m < MT; ++m) s[m][0] = s[m][1] = s[m][2] = s[m][3] = 0.f;
        const uint32_t kaddr = ts + ((warp * 8 + (lane & 7)) * pitch + (lane >> 3) * 8) * 2;
        const uint32_t qaddr = smem_u32(qs) + ((lane & 15) * pitch + (lane >> 4) * 8) * 2;
#pragma unroll 3
        for (uint32_t k = 0; k < ks; ++k) {                                // 32 elements of the rows per step
            uint32_t f[4];
            ldmatrix4(f, kaddr + 64 * k);
#pragma unroll
            for (int m = 0; m < MT; ++m) {
                uint32_t q0[4], q1[4];
                ldmatrix4(q0, qaddr + (16 * m * pitch) * 2 + 64 * k);
                ldmatrix4(q1, qaddr + (16 * m * pitch) * 2 + 64 * k + 32);
                mma_bf16(s[m], q0, f[0], f[1]);
                mma_bf16(s[m], q1, f[2], f[3]);
            }
        }
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const uint32_t key = warp * 8 + 2 * t4 + (i & 1);
                sc[(16 * m + gid + 8 * (i >> 1)) * LT_SP + key] = key < cnt ? s[m][i] * a.scale : -CUDART_INF_F;
            }
        __syncthreads();
#pragma unroll
        for (int g = 0; g < HW; ++g) {
            const uint32_t h = warp * HW + g;
            const float s0 = sc[h * LT_SP + lane], s1 = sc[h * LT_SP + 32 + lane];
            float bm = fmaxf(s0, s1);
#pragma unroll
            for (int d = 16; d > 0; d >>= 1) bm = fmaxf(bm, __shfl_xor_sync(0xffffffffu, bm, d));
            const float nm = fmaxf(mx[g], bm), c = expf(mx[g] - nm), e0 = expf(s0 - nm), e1 = expf(s1 - nm);      // (key p0 is always seen: nm is finite)
            l[g] = l[g] * c + warp_sum(e0 + e1);
            mx[g] = nm;
            ps[h * LT_PP + lane] = __float2bfloat16_rn(e0);
            ps[h * LT_PP + 32 + lane] = __float2bfloat16_rn(e1);
            if (lane == 0) corr[h] = c;
        }
        __syncthreads();
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            const float c0 = corr[16 * m + gid], c1 = corr[16 * m + gid + 8];
#pragma unroll
            for (int c = 0; c < NT; ++c) { o[m][c][0] *= c0; o[m][c][1] *= c0; o[m][c][2] *= c1; o[m][c][3] *= c1; }
        }
#pragma unroll
        for (int k = 0; k < static_cast<int>(LT_KEYS) / 16; ++k) {
            uint32_t pa[MT][4];
#pragma unroll
            for (int m = 0; m < MT; ++m) ldmatrix4(pa[m], smem_u32(ps) + ((16 * m + (lane & 15)) * LT_PP + 16 * k + (lane >> 4) * 8) * 2);
#pragma unroll
            for (int c = 0; c < NT; c += 2) {
                if (col0 + 8 * c >= rp) continue;
                uint32_t f[4];
                ldmatrix4_trans(f, ts + ((16 * k + ((lane >> 3) & 1) * 8 + (lane & 7)) * pitch + col0 + 8 * c + (lane >> 4) * 8) * 2);
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    mma_bf16(o[m][c], pa[m], f[0], f[1]);
                    mma_bf16(o[m][c + 1], pa[m], f[2], f[3]);
                }
            }
        }
        __syncthreads();
        if (bufs == 2) b ^= 1;
        else if (p0 + LT_KEYS < hi) stage(p0 + LT_KEYS, 0);
    }
    // this split's sums and statistics to shared memory (over the tiles, which nobody reads any more)
    float* sums = reinterpret_cast<float*>(tile);                          // [HG][rp]
#pragma unroll
    for (int g = 0; g < HW; ++g)
        if (lane == 0) { stats[warp * HW + g][0] = mx[g]; stats[warp * HW + g][1] = l[g]; }
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int c = 0; c < NT; ++c)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const uint32_t d = col0 + 8 * c + 2 * t4;
                if (d < rp) *reinterpret_cast<float2*>(sums + (16 * m + gid + 8 * u) * rp + d) = make_float2(o[m][c][2 * u], o[m][c][2 * u + 1]);
            }
    namespace cg = cooperative_groups;
    const cg::cluster_group cl = cg::this_cluster();
    const uint32_t rank = cl.block_rank(), size = cl.num_blocks();
    cl.sync();
    float* dst = part + (static_cast<size_t>(split / size) * a.heads + h_cta) * part_elems(a);
    if (threadIdx.x < HG) {
        const uint32_t h = threadIdx.x;
        float m = -CUDART_INF_F, t = 0.f;
        for (uint32_t r = 0; r < size; ++r) m = fmaxf(m, cl.map_shared_rank(&stats[0][0], r)[2 * h]);
        for (uint32_t r = 0; r < size; ++r) {
            const float* st = cl.map_shared_rank(&stats[0][0], r) + 2 * h;
            const float c = st[0] == -CUDART_INF_F ? 0.f : expf(st[0] - m);
            weight[r][h] = c;
            t += st[1] * c;
        }
        if (rank == 0 && h_cta + h < a.heads) { dst[h * part_elems(a)] = m; dst[h * part_elems(a) + 1] = t; }
    }
    __syncthreads();
    for (uint32_t i = rank * LD_WARPS * 32 + threadIdx.x; i < HG * (rp / 4); i += size * LD_WARPS * 32) {
        const uint32_t h = i / (rp / 4), d = 4 * (i % (rp / 4));
        if (h_cta + h >= a.heads) break;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (uint32_t r = 0; r < LT_CLUSTER; ++r) {
            if (r >= size) break;
            const float4 x = *reinterpret_cast<const float4*>(cl.map_shared_rank(sums, r) + h * rp + d);
            axpy(v, weight[r][h], x);
        }
        *reinterpret_cast<float4*>(dst + h * part_elems(a) + 4 + d) = v;
    }
    cl.sync();                                                             // nobody leaves while its sums are read
}

// grid (heads, slices of the value rows): merge of the splits, then the head's value matrix
constexpr uint32_t LD_SPLITS = 64, LO_ROWS = 32, LD_RANK = 1024;
__global__ void __launch_bounds__(256) latent_out_kernel(const __grid_constant__ hf2q_latent_attn a, uint32_t nsplit, const float* __restrict__ part,
                                                         float* __restrict__ out) {
    __shared__ __align__(16) float o[LD_RANK];
    __shared__ float w[LD_SPLITS];
    pdl_trigger();
    {
        const uint32_t v0 = min(blockIdx.y * LO_ROWS, a.vdim), bytes = min(LO_ROWS, a.vdim - v0) * pad8(a.kv_rank) * 2;
        const char* u = static_cast<const char*>(a.uv) + (static_cast<size_t>(blockIdx.x) * a.vdim + v0) * pad8(a.kv_rank) * 2;
        for (uint32_t i = 128 * threadIdx.x; i < bytes; i += 128 * 256) prefetch_l2(u + i);
    }
    pdl_wait();
    const uint32_t h = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, rp = pad8(a.kv_rank);
    const size_t step = static_cast<size_t>(a.heads) * part_elems(a);
    const float* src = part + static_cast<size_t>(h) * part_elems(a);
    if (warp == 0) {
        float m = -CUDART_INF_F, l = 0.f;
        for (uint32_t k = lane; k < nsplit; k += 32) m = fmaxf(m, src[k * step]);
#pragma unroll
        for (int d = 16; d > 0; d >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, d));
        for (uint32_t k = lane; k < nsplit; k += 32) {
            const float mk = src[k * step], c = mk == -CUDART_INF_F ? 0.f : expf(mk - m);
            w[k] = c;
            l += src[k * step + 1] * c;
        }
        l = warp_sum(l);
        for (uint32_t k = lane; k < nsplit; k += 32) w[k] /= l;
    }
    __syncthreads();
    for (uint32_t i = threadIdx.x; i < rp; i += 256) {
        float s = 0.f;
#pragma unroll 8
        for (uint32_t k = 0; k < nsplit; ++k) s = fmaf(w[k], src[k * step + 4 + i], s);
        o[i] = s;
    }
    __syncthreads();
    const uint32_t v1 = min((blockIdx.y + 1) * LO_ROWS, a.vdim);
    for (uint32_t v = blockIdx.y * LO_ROWS + warp; v < v1; v += 8) {
        const __nv_bfloat16* r = static_cast<const __nv_bfloat16*>(a.uv) + (static_cast<size_t>(h) * a.vdim + v) * rp;
        float s = 0.f;
#pragma unroll 2
        for (uint32_t c = 8 * lane; c < rp; c += 256) {
            float f[8];
            load8(r + c, f);
#pragma unroll
            for (int i = 0; i < 8; ++i) s = fmaf(f[i], o[c + i], s);
        }
        s = warp_sum(s);
        if (lane == 0) out[h * a.vdim + v] = s;
    }
}

// ---------------------------------------------------------------- host side
bool latent_ok(const hf2q_latent_attn* a) {
    return a && a->proj && a->norm && a->freq && a->cache && a->pos && a->heads && a->dim && a->dim <= LD_DIM && a->rot_dim && 2 * a->rot_pairs <= a->rot_dim &&
           a->vdim && a->kv_rank && a->kv_rank <= LD_RANK && a->window && a->capacity >= a->window && (a->cache_dtype == HF2Q_DT_F32 || a->cache_dtype == HF2Q_DT_BF16) &&
           reinterpret_cast<uintptr_t>(a->cache) % 16 == 0;
}
constexpr size_t LD_SMEM = 220 * 1024;
size_t decode_smem(const hf2q_latent_attn& a, uint32_t nh, uint32_t elem) {
    return static_cast<size_t>(LD_WARPS) * nh * row_elems(a) * 4 + 2ull * LD_KEYS * (row_elems(a) + 16 / elem) * elem;
}
uint32_t elem_bytes(const hf2q_latent_attn& a) { return a.cache_dtype == HF2Q_DT_F32 ? 4 : 2; }
uint32_t heads_per_warp(const hf2q_latent_attn& a) {
    return a.heads > 2 * LD_WARPS && a.kv_rank <= 512 && decode_smem(a, 4, elem_bytes(a)) <= LD_SMEM ? 4 : 1;
}
size_t mma_smem(const hf2q_latent_attn& a, uint32_t mt, uint32_t bufs) {
    return 16ull * mt * (tile_pitch(a) * 2 + LT_SP * 4 + LT_PP * 2) + static_cast<size_t>(bufs) * LT_KEYS * tile_pitch(a) * 2;
}
// 16 heads per CTA as long as the tiles of the window do not fill the GPU
uint32_t mma_mt(const hf2q_latent_attn& a, int sms) {
    const uint64_t ctas = static_cast<uint64_t>((a.heads + 15) / 16) * ((a.window + LT_KEYS - 1) / LT_KEYS);
    return a.heads > 16 && ctas > static_cast<uint64_t>(sms) && mma_smem(a, 2, 1) <= LD_SMEM ? 2 : 1;
}
bool on_tensor_cores(const hf2q_latent_attn& a) { return a.cache_dtype == HF2Q_DT_BF16 && a.kv_rank <= 512 && mma_smem(a, 1, 1) <= LD_SMEM; }
uint32_t head_groups(const hf2q_latent_attn& a, int sms) {
    const uint32_t per = on_tensor_cores(a) ? 16 * mma_mt(a, sms) : LD_WARPS * heads_per_warp(a);
    return (a.heads + per - 1) / per;
}
uint32_t cluster_of(uint32_t splits) { return splits % 8 == 0 ? 8 : splits % 4 == 0 ? 4 : splits % 2 == 0 ? 2 : 1; }
uint32_t decode_splits(const hf2q_latent_attn& a, int sms) {
    const bool tc = on_tensor_cores(a);
    const uint32_t keys = tc ? LT_KEYS : LD_KEYS, by_sm = static_cast<uint32_t>(sms) / head_groups(a, sms), by_keys = (a.window + keys - 1) / keys;
    uint32_t s = by_sm < by_keys ? by_sm : by_keys;
    s = s < 1 ? 1 : s > LD_SPLITS ? LD_SPLITS : s;
    return tc && s > 8 ? s / 8 * 8 : s;                                    // whole clusters
}
uint64_t query_floats(const hf2q_latent_attn& a) { return (static_cast<uint64_t>(a.heads) * row_elems(a) + 63) & ~63ull; }

template <typename T, int NH, int NC>
cudaError_t launch_decode(const hf2q_latent_attn& a, const float* qa, float* part, uint32_t splits, uint32_t groups, cudaStream_t st) {
    static PerDeviceFlag flag;
    if (const cudaError_t e = ensure_max_dynamic_smem(latent_decode_kernel<T, NH, NC>, static_cast<int>(LD_SMEM), flag); e != cudaSuccess) return e;
    const uint32_t bufs = decode_smem(a, NH, sizeof(T)) <= LD_SMEM ? 2 : 1;
    const size_t smem = decode_smem(a, NH, sizeof(T)) - (bufs == 1 ? static_cast<size_t>(LD_KEYS) * (row_elems(a) + 16 / sizeof(T)) * sizeof(T) : 0);
    if (smem > LD_SMEM) return cudaErrorInvalidValue;
    return launch_pdl(latent_decode_kernel<T, NH, NC>, dim3(groups, splits), dim3(LD_WARPS * 32), smem, st, a, bufs, qa, part);
}
template <int MT, int NT>
cudaError_t launch_decode_nt(const hf2q_latent_attn& a, const float* qa, float* part, uint32_t splits, uint32_t groups, cudaStream_t st) {
    static PerDeviceFlag flag;
    if (const cudaError_t e = ensure_max_dynamic_smem(latent_decode_mma_kernel<MT, NT>, static_cast<int>(LD_SMEM), flag); e != cudaSuccess) return e;
    const uint32_t tiles = (a.window + LT_KEYS - 1) / LT_KEYS, bufs = tiles > splits && mma_smem(a, MT, 2) <= LD_SMEM ? 2 : 1;
    return launch_pdl_cluster(latent_decode_mma_kernel<MT, NT>, dim3(groups, splits), dim3(LD_WARPS * 32), dim3(1, cluster_of(splits)), mma_smem(a, MT, bufs), st, a, bufs,
                              qa, part);
}
template <int MT>
cudaError_t launch_decode_mma(const hf2q_latent_attn& a, const float* qa, float* part, uint32_t splits, uint32_t groups, cudaStream_t st) {
    if (a.kv_rank <= 128) return launch_decode_nt<MT, 2>(a, qa, part, splits, groups, st);
    if (a.kv_rank <= 256) return launch_decode_nt<MT, 4>(a, qa, part, splits, groups, st);
    return launch_decode_nt<MT, 8>(a, qa, part, splits, groups, st);
}
template <typename T>
cudaError_t launch_decode_any(const hf2q_latent_attn& a, const float* qa, float* part, uint32_t splits, uint32_t groups, int sms, cudaStream_t st) {
    if (on_tensor_cores(a)) return mma_mt(a, sms) == 2 ? launch_decode_mma<2>(a, qa, part, splits, groups, st) : launch_decode_mma<1>(a, qa, part, splits, groups, st);
    if (heads_per_warp(a) == 4) {
        if (a.kv_rank <= 128) return launch_decode<T, 4, 2>(a, qa, part, splits, groups, st);
        return launch_decode<T, 4, 8>(a, qa, part, splits, groups, st);
    }
    if (a.kv_rank <= 128) return launch_decode<T, 1, 2>(a, qa, part, splits, groups, st);
    if (a.kv_rank <= 512) return launch_decode<T, 1, 8>(a, qa, part, splits, groups, st);
    return launch_decode<T, 1, 16>(a, qa, part, splits, groups, st);
}

}  // namespace
}  // namespace hf2q

using namespace hf2q;
using namespace hf2q::seq;

extern "C" {

HF2Q_API int32_t hf2q_cuda_latent_scratch_bytes(hf2q_ctx* ctx, const hf2q_latent_attn* a, uint64_t* out) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!a || !out || a->heads == 0 || a->kv_rank == 0 || a->window == 0) return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "latent_scratch_bytes: bad sizes");
    *out = 4 * (query_floats(*a) + static_cast<uint64_t>(decode_splits(*a, ctx_sm_count(ctx))) * a->heads * part_elems(*a));
    return HF2Q_OK;
}

HF2Q_API int32_t hf2q_cuda_latent_decode(hf2q_ctx* ctx, void* stream, const hf2q_latent_attn* a, float* out, void* scratch, uint64_t scratch_bytes) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    uint64_t need = 0;
    if (!latent_ok(a) || !a->uk_t || !a->uv || !out || !scratch || (reinterpret_cast<uintptr_t>(a->uk_t) | reinterpret_cast<uintptr_t>(a->uv) | reinterpret_cast<uintptr_t>(scratch)) % 16 ||
        hf2q_cuda_latent_scratch_bytes(ctx, a, &need) != HF2Q_OK)
        return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "latent_decode: null or unaligned pointer, or an unsupported size");
    if (scratch_bytes < need) return ctx_fail(ctx, HF2Q_ERR_WORKSPACE, "latent_decode: scratch too small");
    const cudaStream_t st = static_cast<cudaStream_t>(stream);
    float* qa = static_cast<float*>(scratch);
    float* part = qa + query_floats(*a);
    const int sms = ctx_sm_count(ctx);
    const uint32_t splits = decode_splits(*a, sms), groups = head_groups(*a, sms), parts = on_tensor_cores(*a) ? splits / cluster_of(splits) : splits, slices = (pad8(a->kv_rank) + LQ_ROWS - 1) / LQ_ROWS;
    const dim3 grid_q(a->heads * slices + 1);
    const bool f32 = a->cache_dtype == HF2Q_DT_F32;
    cudaError_t e = f32 ? launch_pdl(latent_query_kernel<float>, grid_q, dim3(256), 0, st, *a, slices, qa)
                        : launch_pdl(latent_query_kernel<__nv_bfloat16>, grid_q, dim3(256), 0, st, *a, slices, qa);
    if (e == cudaSuccess) e = f32 ? launch_decode_any<float>(*a, qa, part, splits, groups, sms, st) : launch_decode_any<__nv_bfloat16>(*a, qa, part, splits, groups, sms, st);
    if (e == cudaSuccess) e = launch_pdl(latent_out_kernel, dim3(a->heads, (a->vdim + LO_ROWS - 1) / LO_ROWS), dim3(256), 0, st, *a, parts, part, out);
    return ctx_cuda_result(ctx, e, "latent_decode", 3);
}

HF2Q_API int32_t hf2q_cuda_latent_append(hf2q_ctx* ctx, void* stream, const hf2q_latent_attn* a, uint32_t m, void* q_out) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!latent_ok(a) || !q_out || a->window - 1 + static_cast<uint64_t>(m) > a->capacity)
        return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "latent_append: null pointer, an unsupported size or more tokens than the ring holds");
    if (m == 0) return HF2Q_OK;
    const dim3 grid(static_cast<unsigned>((static_cast<uint64_t>(m) * (a->heads + 1) + 7) / 8));
    const cudaStream_t st = static_cast<cudaStream_t>(stream);
    const cudaError_t e = a->cache_dtype == HF2Q_DT_F32 ? launch_pdl(latent_append_kernel<float>, grid, dim3(256), 0, st, *a, m, static_cast<float*>(q_out))
                                                        : launch_pdl(latent_append_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, *a, m, static_cast<__nv_bfloat16*>(q_out));
    return ctx_cuda_result(ctx, e, "latent_append", 1);
}

}  // extern "C"
