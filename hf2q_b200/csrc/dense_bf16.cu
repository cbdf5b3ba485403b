// Products with bf16 weights: y[m][n] = epilogue(x[m][k] . w[n][k]^T), f32 accumulation.
//
//   dense_matvec_kernel   m = 1..8 rows; weights streamed with 16-byte loads, activations f32 in shared memory, fp32
//                         arithmetic (HBM-bound: 2 bytes per weight against one FMA per row).  With one row the
//                         layer's norm / token shift / gating runs in the kernel's own prologue.
//   dense_gemm_tc_kernel  more rows, bf16 activations: persistent tcgen05 kernel, both operands by TMA with 128-byte
//                         swizzle, two accumulator buffers in tensor memory so that the epilogue of a tile runs under
//                         the main loop of the next.
//   dense_gemm_f32_kernel more rows, f32 activations: CUDA-core tiles in full 32-bit arithmetic.
#include "seq_common.cuh"
#include "tc_common.cuh"

namespace hf2q {
namespace {
using namespace seq;

__device__ __forceinline__ float epilogue_value(float v, uint32_t epi, float cap) {
    if (epi == HF2Q_EPI_GELU) return gelu_tanhf(v);
    if (epi == HF2Q_EPI_SOFTCAP) return cap * tanhf(v / cap);
    return v;
}

// ---------------------------------------------------------------- mat-vec
constexpr int MV_WARPS = 8;
constexpr int MV_THREADS = MV_WARPS * 32;

// acc[r][m] += w rows (row0 + r) . xs rows; one warp, RW weight rows, 8 elements per lane and step
template <int RW, int M>
__device__ __forceinline__ void matvec_rows(const __nv_bfloat16* __restrict__ w, uint32_t row0, uint32_t n, uint32_t k, const float* xs,
                                            float (&acc)[RW][M]) {
    const uint32_t lane = threadIdx.x & 31;
    const uint4* wr[RW];
#pragma unroll
    for (int r = 0; r < RW; ++r) wr[r] = reinterpret_cast<const uint4*>(w + static_cast<size_t>(min(row0 + r, n - 1)) * k);
    const uint32_t steps = k / 8;
    auto take = [&](const uint4& v, int r, uint32_t c) {
        const float f[8] = {bf_lo(v.x), bf_hi(v.x), bf_lo(v.y), bf_hi(v.y), bf_lo(v.z), bf_hi(v.z), bf_lo(v.w), bf_hi(v.w)};
#pragma unroll
        for (int m = 0; m < M; ++m) {
            const float4 a = *reinterpret_cast<const float4*>(xs + static_cast<size_t>(m) * k + 8 * c);
            const float4 b = *reinterpret_cast<const float4*>(xs + static_cast<size_t>(m) * k + 8 * c + 4);
            float s = acc[r][m];
            s = fmaf(f[0], a.x, s); s = fmaf(f[1], a.y, s); s = fmaf(f[2], a.z, s); s = fmaf(f[3], a.w, s);
            s = fmaf(f[4], b.x, s); s = fmaf(f[5], b.y, s); s = fmaf(f[6], b.z, s); s = fmaf(f[7], b.w, s);
            acc[r][m] = s;
        }
    };
    constexpr int U = 4;
    uint32_t c = lane;
    for (; c + 32 * (U - 1) < steps; c += 32 * U) {
        uint4 v[U][RW];
#pragma unroll
        for (int u = 0; u < U; ++u)
#pragma unroll
            for (int r = 0; r < RW; ++r) v[u][r] = __ldcs(wr[r] + c + 32 * u);
#pragma unroll
        for (int u = 0; u < U; ++u)
#pragma unroll
            for (int r = 0; r < RW; ++r) take(v[u][r], r, c + 32 * u);
    }
    for (; c < steps; c += 32) {
#pragma unroll
        for (int r = 0; r < RW; ++r) take(__ldcs(wr[r] + c), r, c);
    }
#pragma unroll
    for (int r = 0; r < RW; ++r)
#pragma unroll
        for (int m = 0; m < M; ++m) acc[r][m] = warp_sum(acc[r][m]);
}

struct MatvecSegs {
    hf2q_matvec s[2];
    uint32_t blocks0;        // CTAs of segment 0
};

// One-row product.  A CTA owns a contiguous range of weight rows, cut into chunks of MV_CHUNK elements; its warps take
// the chunks in turn, each through a private ring of bulk copies that starts filling before the wait for the previous
// kernel (weights never change).  Chunk sums of a block of rows meet in shared memory and are added in chunk order.
constexpr int MR_WARPS = 16, MR_THREADS = MR_WARPS * 32, MV_CHUNK = 1024, MR_STAGES = 3, MR_PART = 2048;
constexpr uint32_t MR_RING = MR_WARPS * MR_STAGES * MV_CHUNK * 2;

template <int PRO>
__global__ void __launch_bounds__(MR_THREADS) dense_matvec_kernel(const __grid_constant__ MatvecSegs p, uint32_t* status) {
    extern __shared__ __align__(128) uint8_t mv_smem[];                 // ring, then x [k] f32
    __shared__ float red[64];
    __shared__ float part[2][MR_PART];
    __shared__ uint64_t bars[MR_WARPS][MR_STAGES];
    pdl_trigger();
    const bool second = blockIdx.x >= p.blocks0;
    const hf2q_matvec& s = p.s[second];
    const uint32_t blk = blockIdx.x - (second ? p.blocks0 : 0u), n_blk = second ? gridDim.x - p.blocks0 : p.blocks0;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    __nv_bfloat16* ring = reinterpret_cast<__nv_bfloat16*>(mv_smem) + static_cast<size_t>(warp) * MR_STAGES * MV_CHUNK;
    float* xs = reinterpret_cast<float*>(mv_smem + MR_RING);
    // rows [row0, row1) of this CTA, spread evenly
    const uint32_t row0 = static_cast<uint32_t>(static_cast<uint64_t>(s.n) * blk / n_blk), row1 = static_cast<uint32_t>(static_cast<uint64_t>(s.n) * (blk + 1) / n_blk);
    const uint32_t per_row = (s.k + MV_CHUNK - 1) / MV_CHUNK, n_chunks = (row1 - row0) * per_row;
    const __nv_bfloat16* w = static_cast<const __nv_bfloat16*>(s.w) + static_cast<size_t>(row0) * s.k;
    auto issue = [&](uint32_t i) {                                      // this warp's chunk number i
        const uint32_t c = i * MR_WARPS + warp;
        if (c >= n_chunks) return;
        const uint32_t k0 = (c % per_row) * MV_CHUNK, bytes = min(static_cast<uint32_t>(MV_CHUNK), s.k - k0) * 2;
        uint64_t* bar = &bars[warp][i % MR_STAGES];
        mbar_arrive_expect_tx(bar, bytes);
        bulk_g2s(ring + (i % MR_STAGES) * MV_CHUNK, w + static_cast<size_t>(c / per_row) * s.k + k0, bytes, bar);
    };
    if (lane == 0) {
        for (int i = 0; i < MR_STAGES; ++i) mbar_init(&bars[warp][i], 1);
        mbar_fence_init();
        for (int i = 0; i < MR_STAGES; ++i) issue(i);
    }
    pdl_wait();
    if constexpr (PRO == HF2Q_PRO_NONE) {
        for (uint32_t i = threadIdx.x; i < s.k; i += MR_THREADS) xs[i] = s.x[i];
    } else if constexpr (PRO == HF2Q_PRO_NORM) {
        const hf2q_pre_norm& q = s.pre;
        const float inv = residual_row(q, 0, xs, red);
        const bool keep = blk == 0;
        const uint32_t pos = q.shift ? *q.pos : 0u;
        const float* before = q.shift_state + static_cast<size_t>((pos + 1) & 1) * q.width;
        float* now = q.shift_state + static_cast<size_t>(pos & 1) * q.width;
        for (uint32_t i = threadIdx.x; i < s.k; i += MR_THREADS) {
            float h = 0.f;
            if (i < q.width) {
                const float x = xs[i];
                if (keep && q.x_out) q.x_out[i] = x;
                h = x * inv * q.norm[i];
                if (q.shift) {
                    if (keep) now[i] = h;
                    h += (before[i] - h) * q.shift[i];
                }
            }
            xs[i] = h;
        }
    } else {
        for (uint32_t i = s.gated.heads * s.gated.head_dim + threadIdx.x; i < s.k; i += MR_THREADS) xs[i] = 0.f;
        gated_heads_row<float>(s.gated, 0, xs, warp, MR_WARPS);
    }
    __syncthreads();
    const uint32_t block_rows = max(1u, MR_PART / per_row);
    bool ok = true;
    uint32_t i = 0;                                                     // this warp's chunk counter
    for (uint32_t r0 = 0, pb = 0; r0 < row1 - row0; r0 += block_rows, pb ^= 1) {
        const uint32_t rows = min(block_rows, row1 - row0 - r0), c_end = (r0 + rows) * per_row;
        for (uint32_t c = i * MR_WARPS + warp; c < c_end; ++i, c += MR_WARPS) {
            const uint32_t st = i % MR_STAGES, kc = c % per_row, k0 = kc * MV_CHUNK, len = min(static_cast<uint32_t>(MV_CHUNK), s.k - k0);
            if (ok) ok = mbar_wait_bounded(&bars[warp][st], (i / MR_STAGES) & 1, status);
            ok = __all_sync(0xffffffffu, ok);
            float acc = 0.f;
            if (ok) {
                const uint4* wv = reinterpret_cast<const uint4*>(ring + st * MV_CHUNK);
                const float* xv = xs + k0;
#pragma unroll
                for (int u = 0; u < MV_CHUNK / 256; ++u) {
                    const uint32_t e = lane + 32 * u;
                    if (8 * e < len) {
                        const uint4 v = wv[e];
                        const float4 a = *reinterpret_cast<const float4*>(xv + 8 * e), b = *reinterpret_cast<const float4*>(xv + 8 * e + 4);
                        acc = fmaf(bf_lo(v.x), a.x, acc); acc = fmaf(bf_hi(v.x), a.y, acc); acc = fmaf(bf_lo(v.y), a.z, acc); acc = fmaf(bf_hi(v.y), a.w, acc);
                        acc = fmaf(bf_lo(v.z), b.x, acc); acc = fmaf(bf_hi(v.z), b.y, acc); acc = fmaf(bf_lo(v.w), b.z, acc); acc = fmaf(bf_hi(v.w), b.w, acc);
                    }
                }
            }
            __syncwarp();                                               // every lane has read the stage
            if (lane == 0 && ok) issue(i + MR_STAGES);
            acc = warp_sum(acc);
            if (lane == 0) part[pb][c - r0 * per_row] = acc;
        }
        __syncthreads();                                                // (the other half of `part` is free: its readers passed this barrier)
        for (uint32_t r = threadIdx.x; r < rows; r += MR_THREADS) {
            float v = 0.f;
            for (uint32_t kc = 0; kc < per_row; ++kc) v += part[pb][r * per_row + kc];
            const uint32_t row = row0 + r0 + r;
            v = epilogue_value(v, s.epilogue, s.cap);
            if (s.epilogue == HF2Q_EPI_ADD) v += s.residual[row];
            s.y[row] = v;
        }
    }
}

struct DenseArgs {
    const void* x;
    const __nv_bfloat16* w;
    void* y;
    const float* residual;
    uint32_t ldx, ldy, m, n, k, epi;
    float cap;
};

template <typename X, typename Y, int M>
__global__ void __launch_bounds__(MV_THREADS) dense_matvec_m_kernel(const DenseArgs p) {
    extern __shared__ __align__(16) float xs[];
    pdl_trigger();
    pdl_wait();
    const X* x = static_cast<const X*>(p.x);
    for (int m = 0; m < M; ++m)
        for (uint32_t i = threadIdx.x; i < p.k; i += MV_THREADS)
            xs[static_cast<size_t>(m) * p.k + i] = m < static_cast<int>(p.m) ? to_f32(x[static_cast<size_t>(m) * p.ldx + i]) : 0.f;
    __syncthreads();
    const uint32_t row = blockIdx.x * MV_WARPS + (threadIdx.x >> 5);
    if (row >= p.n) return;
    float acc[1][M];
#pragma unroll
    for (int m = 0; m < M; ++m) acc[0][m] = 0.f;
    matvec_rows<1, M>(p.w, row, p.n, p.k, xs, acc);
    if ((threadIdx.x & 31) == 0) {
#pragma unroll
        for (int m = 0; m < M; ++m)
            if (m < static_cast<int>(p.m)) {
                const size_t o = static_cast<size_t>(m) * p.ldy + row;
                float v = epilogue_value(acc[0][m], p.epi, p.cap);
                if (p.epi == HF2Q_EPI_ADD) v += p.residual[o];
                static_cast<Y*>(p.y)[o] = from_f32<Y>(v);
            }
    }
}

// ---------------------------------------------------------------- fp32 product on the CUDA cores
constexpr int FT = 64, FK = 16;

template <typename X, typename Y>
__global__ void __launch_bounds__(256) dense_gemm_f32_kernel(const DenseArgs p) {
    __shared__ float as[FK][FT + 4], bs[FK][FT + 4];
    pdl_trigger();
    pdl_wait();
    const X* x = static_cast<const X*>(p.x);
    const uint32_t m0 = blockIdx.y * FT, n0 = blockIdx.x * FT;
    const uint32_t tr = threadIdx.x / 16, tc = threadIdx.x % 16;
    float acc[4][4] = {};
    for (uint32_t k0 = 0; k0 < p.k; k0 += FK) {
        for (uint32_t i = threadIdx.x; i < FT * FK; i += 256) {
            const uint32_t r = i / FK, c = i % FK;
            as[c][r] = m0 + r < p.m && k0 + c < p.k ? to_f32(x[static_cast<size_t>(m0 + r) * p.ldx + k0 + c]) : 0.f;
            bs[c][r] = n0 + r < p.n && k0 + c < p.k ? to_f32(p.w[static_cast<size_t>(n0 + r) * p.k + k0 + c]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int c = 0; c < FK; ++c) {
            const float4 a = *reinterpret_cast<const float4*>(&as[c][4 * tr]), b = *reinterpret_cast<const float4*>(&bs[c][4 * tc]);
            const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
        }
        __syncthreads();
    }
    for (int i = 0; i < 4; ++i)
        for (int j = 0; j < 4; ++j) {
            const uint32_t r = m0 + 4 * tr + i, c = n0 + 4 * tc + j;
            if (r >= p.m || c >= p.n) continue;
            const size_t o = static_cast<size_t>(r) * p.ldy + c;
            float v = epilogue_value(acc[i][j], p.epi, p.cap);
            if (p.epi == HF2Q_EPI_ADD) v += p.residual[o];
            static_cast<Y*>(p.y)[o] = from_f32<Y>(v);
        }
}

// ---------------------------------------------------------------- tcgen05 product
// One CTA per SM walks tiles of 128 activation rows x NT weight rows.  Warp 0: TMA producer; warp 1: tensor-memory
// owner and MMA issuer; warps 2..5: epilogue (thread = activation row).
constexpr int TC_M = 128, TC_K = 64, TC_THREADS = 192;
__host__ __device__ constexpr int tc_stages(int nt) { return nt == 256 ? 4 : nt == 128 ? 6 : 8; }
__host__ __device__ constexpr uint32_t tc_stage_bytes(int nt) { return (TC_M + nt) * TC_K * 2; }

__device__ __forceinline__ void umma_ss(uint32_t d, uint64_t a, uint64_t b, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
        ::"r"(d), "l"(a), "l"(b), "r"(idesc), "r"(accumulate)
        : "memory");
}
__device__ __forceinline__ void st_global_v8(float* p, const float* v) {
    asm volatile("st.global.v8.f32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8};" ::"l"(p), "f"(v[0]), "f"(v[1]), "f"(v[2]), "f"(v[3]), "f"(v[4]), "f"(v[5]),
                 "f"(v[6]), "f"(v[7])
                 : "memory");
}

template <int NT, typename Y>
__global__ void __launch_bounds__(TC_THREADS, 1) dense_gemm_tc_kernel(const __grid_constant__ CUtensorMap map_x, const __grid_constant__ CUtensorMap map_w,
                                                                      const DenseArgs p, uint32_t* status) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
    constexpr int ST = tc_stages(NT);
    constexpr uint32_t SB = tc_stage_bytes(NT);
    __shared__ uint64_t full[ST], empty[ST], d_full[2], d_empty[2];
    __shared__ uint32_t tmem_slot;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t mt = (p.m + TC_M - 1) / TC_M, n_tiles = mt * ((p.n + NT - 1) / NT), nkb = (p.k + TC_K - 1) / TC_K;
    if (threadIdx.x == 0) {
        for (int i = 0; i < ST; ++i) { mbar_init(&full[i], 1); mbar_init(&empty[i], 1); }
        for (int i = 0; i < 2; ++i) { mbar_init(&d_full[i], 1); mbar_init(&d_empty[i], 4); }
        mbar_fence_init();
    }
    if (warp == 1) { tc::tmem_alloc(&tmem_slot, 2 * NT); tc::tmem_relinquish(); }
    tc::tc_fence_before();
    __syncthreads();
    tc::tc_fence_after();
    const uint32_t tmem = tmem_slot;
    pdl_trigger();
    pdl_wait();
    if (warp == 0) {
        if (lane == 0) {
            uint32_t it = 0;
            bool ok = true;
            for (uint32_t tile = blockIdx.x; tile < n_tiles && ok; tile += gridDim.x) {
                const int row_x = static_cast<int>((tile % mt) * TC_M), row_w = static_cast<int>((tile / mt) * NT);
                for (uint32_t kb = 0; kb < nkb; ++kb, ++it) {
                    const uint32_t s = it % ST;
                    if (it >= ST) ok = mbar_wait_bounded(&empty[s], (it / ST - 1) & 1, status);
                    if (!ok) break;
                    mbar_arrive_expect_tx(&full[s], SB);
                    tc::tma_2d(smem + s * SB, &map_x, static_cast<int>(kb * TC_K), row_x, &full[s]);
                    tc::tma_2d(smem + s * SB + TC_M * TC_K * 2, &map_w, static_cast<int>(kb * TC_K), row_w, &full[s]);
                }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            // D f32, A and B bf16, both K-major, M = 128, N = NT
            constexpr uint32_t IDESC = (1u << 4) | (1u << 7) | (1u << 10) | (static_cast<uint32_t>(NT >> 3) << 17) | (static_cast<uint32_t>(TC_M >> 4) << 24);
            uint32_t it = 0, li = 0;
            bool ok = true;
            for (uint32_t tile = blockIdx.x; tile < n_tiles && ok; tile += gridDim.x, ++li) {
                const uint32_t b = li & 1;
                if (li >= 2) ok = mbar_wait_bounded(&d_empty[b], (li / 2 - 1) & 1, status);
                if (!ok) break;
                tc::tc_fence_after();
                for (uint32_t kb = 0; kb < nkb; ++kb, ++it) {
                    const uint32_t s = it % ST;
                    ok = mbar_wait_bounded(&full[s], (it / ST) & 1, status);
                    if (!ok) break;
                    tc::tc_fence_after();
                    const uint64_t da = tc::smem_desc_sw128(smem_u32(smem + s * SB)), db = tc::smem_desc_sw128(smem_u32(smem + s * SB + TC_M * TC_K * 2));
#pragma unroll
                    for (uint32_t kk = 0; kk < TC_K / 16; ++kk) umma_ss(tmem + b * NT, da + 2 * kk, db + 2 * kk, IDESC, (kb | kk) ? 1u : 0u);
                    tc::tc_commit(&empty[s]);
                }
                if (ok) tc::tc_commit(&d_full[b]);
            }
        }
    } else {
        const uint32_t quad = warp & 3;
        const bool wide = p.ldy % 8 == 0 && reinterpret_cast<uintptr_t>(p.y) % 32 == 0 &&
                          (p.epi != HF2Q_EPI_ADD || reinterpret_cast<uintptr_t>(p.residual) % 16 == 0);
        uint32_t li = 0;
        for (uint32_t tile = blockIdx.x; tile < n_tiles; tile += gridDim.x, ++li) {
            const uint32_t b = li & 1;
            bool ok = mbar_wait_bounded(&d_full[b], (li / 2) & 1, status);
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) break;
            tc::tc_fence_after();
            const uint32_t row = (tile % mt) * TC_M + quad * 32 + lane, n0 = (tile / mt) * NT;
            const uint32_t n_cols = min(static_cast<uint32_t>(NT), p.n - n0);
#pragma unroll 1
            for (uint32_t c0 = 0; c0 < n_cols; c0 += 32) {
                uint32_t r[32];
                tc::tmem_ld32(tmem + b * NT + ((quad * 32u) << 16) + c0, r);
                tc::tmem_wait_ld();
                if (row < p.m) {
                float v[32];
#pragma unroll
                for (int j = 0; j < 32; ++j) v[j] = __uint_as_float(r[j]);
                const size_t o = static_cast<size_t>(row) * p.ldy + n0 + c0;
                Y* y = static_cast<Y*>(p.y) + o;
                if (p.epi == HF2Q_EPI_GELU || p.epi == HF2Q_EPI_SOFTCAP) {
#pragma unroll
                    for (int j = 0; j < 32; ++j) v[j] = epilogue_value(v[j], p.epi, p.cap);
                }
                if (wide && c0 + 32 <= n_cols) {
                    if (p.epi == HF2Q_EPI_ADD) {
#pragma unroll
                        for (int j = 0; j < 32; j += 4) {
                            const float4 q = *reinterpret_cast<const float4*>(p.residual + o + j);
                            v[j] += q.x; v[j + 1] += q.y; v[j + 2] += q.z; v[j + 3] += q.w;
                        }
                    }
                    if constexpr (sizeof(Y) == 4) {
#pragma unroll
                        for (int j = 0; j < 32; j += 8) st_global_v8(reinterpret_cast<float*>(y) + j, v + j);
                    } else {
                        uint32_t q[16];
#pragma unroll
                        for (int j = 0; j < 16; ++j) {
                            const __nv_bfloat162 h = __floats2bfloat162_rn(v[2 * j], v[2 * j + 1]);
                            q[j] = *reinterpret_cast<const uint32_t*>(&h);
                        }
#pragma unroll
                        for (int j = 0; j < 4; ++j) reinterpret_cast<uint4*>(y)[j] = make_uint4(q[4 * j], q[4 * j + 1], q[4 * j + 2], q[4 * j + 3]);
                    }
                } else {
#pragma unroll
                    for (int j = 0; j < 32; ++j)
                        if (c0 + j < n_cols) {
                            float q = v[j];
                            if (p.epi == HF2Q_EPI_ADD) q += p.residual[o + j];
                            y[j] = from_f32<Y>(q);
                        }
                }
                }
                __syncwarp();
            }
            tc::tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&d_empty[b]);
        }
    }
    tc::tc_fence_before();
    __syncthreads();
    tc::tc_fence_after();
    if (warp == 1) tc::tmem_dealloc(tmem, 2 * NT);
}

// ---------------------------------------------------------------- host side
typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                  const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                  CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
EncodeTiledFn encode_fn() {
    static EncodeTiledFn fn = nullptr;
    static std::once_flag once;
    std::call_once(once, [] {
        void* p = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) == cudaSuccess && q == cudaDriverEntryPointSuccess)
            fn = reinterpret_cast<EncodeTiledFn>(p);
    });
    return fn;
}
// rows x k bf16, `ld` elements between rows; box of 64 elements x box_rows, 128-byte swizzle
bool encode_rows(CUtensorMap* map, const void* base, uint32_t rows, uint32_t k, uint32_t ld, uint32_t box_rows) {
    const EncodeTiledFn fn = encode_fn();
    if (!fn) return false;
    const cuuint64_t dims[2] = {k, rows}, strides[1] = {static_cast<cuuint64_t>(ld) * 2};
    const cuuint32_t box[2] = {TC_K, box_rows}, es[2] = {1, 1};
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
              CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int NT, typename Y>
cudaError_t launch_tc(const DenseArgs& a, int sms, uint32_t* status, cudaStream_t st) {
    CUtensorMap mx, mw;
    if (!encode_rows(&mx, a.x, a.m, a.k, a.ldx, TC_M) || !encode_rows(&mw, a.w, a.n, a.k, a.k, NT)) return cudaErrorInvalidValue;
    const size_t smem = 1024 + static_cast<size_t>(tc_stages(NT)) * tc_stage_bytes(NT);
    static PerDeviceFlag flag;
    if (const cudaError_t e = ensure_max_dynamic_smem(dense_gemm_tc_kernel<NT, Y>, static_cast<int>(smem), flag); e != cudaSuccess) return e;
    const uint32_t tiles = ((a.m + TC_M - 1) / TC_M) * ((a.n + NT - 1) / NT);
    const uint32_t grid = tiles < static_cast<uint32_t>(sms) ? tiles : static_cast<uint32_t>(sms);
    return launch_pdl(dense_gemm_tc_kernel<NT, Y>, dim3(grid), dim3(TC_THREADS), smem, st, mx, mw, a, status);
}
template <typename Y>
cudaError_t launch_tc_any(const DenseArgs& a, int sms, uint32_t* status, cudaStream_t st) {
    const uint32_t mt = (a.m + TC_M - 1) / TC_M;
    // the widest tile that still gives (nearly) every SM work
    if (mt * ((a.n + 255) / 256) >= static_cast<uint32_t>(sms) * 3 / 4) return launch_tc<256, Y>(a, sms, status, st);
    if (mt * ((a.n + 127) / 128) >= static_cast<uint32_t>(sms) * 3 / 4) return launch_tc<128, Y>(a, sms, status, st);
    return launch_tc<64, Y>(a, sms, status, st);
}

constexpr uint32_t MV_SMEM = 200 * 1024;

template <typename X, typename Y, int M>
cudaError_t launch_mv_m(const DenseArgs& a, cudaStream_t st) {
    static PerDeviceFlag flag;
    if (const cudaError_t e = ensure_max_dynamic_smem(dense_matvec_m_kernel<X, Y, M>, MV_SMEM, flag); e != cudaSuccess) return e;
    return launch_pdl(dense_matvec_m_kernel<X, Y, M>, dim3((a.n + MV_WARPS - 1) / MV_WARPS), dim3(MV_THREADS),
                      static_cast<size_t>(M) * a.k * 4, st, a);
}
template <typename X, typename Y>
cudaError_t launch_mv(DenseArgs a, cudaStream_t st, uint64_t* launches) {
    const uint32_t fit = MV_SMEM / (a.k * 4);
    if (fit == 0) return cudaErrorInvalidValue;
    const uint32_t m_total = a.m;
    for (uint32_t m0 = 0; m0 < m_total;) {
        uint32_t step = fit < 8 ? fit : 8;
        if (step > m_total - m0) step = m_total - m0;
        DenseArgs b = a;
        b.m = step;
        b.x = static_cast<const X*>(a.x) + static_cast<size_t>(m0) * a.ldx;
        b.y = static_cast<Y*>(a.y) + static_cast<size_t>(m0) * a.ldy;
        if (a.residual) b.residual = a.residual + static_cast<size_t>(m0) * a.ldy;
        // the smallest kernel that holds `step` rows and fits
        const uint32_t mk = step <= 1 ? 1 : step <= 2 ? 2 : step <= 4 ? 4 : 8;
        cudaError_t e;
        if (mk > fit) { b.m = step = mk / 2; }
        switch (mk > fit ? mk / 2 : mk) {
            case 1: e = launch_mv_m<X, Y, 1>(b, st); break;
            case 2: e = launch_mv_m<X, Y, 2>(b, st); break;
            case 4: e = launch_mv_m<X, Y, 4>(b, st); break;
            default: e = launch_mv_m<X, Y, 8>(b, st); break;
        }
        if (e != cudaSuccess) return e;
        ++*launches;
        m0 += step;
    }
    return cudaSuccess;
}

template <typename X, typename Y>
cudaError_t dense_any(const DenseArgs& a, int sms, uint32_t* status, cudaStream_t st, uint64_t* launches) {
    if (a.m <= 8 && a.k * 4 <= MV_SMEM) return launch_mv<X, Y>(a, st, launches);
    *launches = 1;
    if constexpr (sizeof(X) == 2) {
        if (a.ldx % 8 == 0 && reinterpret_cast<uintptr_t>(a.x) % 16 == 0) return launch_tc_any<Y>(a, sms, status, st);
    }
    return launch_pdl(dense_gemm_f32_kernel<X, Y>, dim3((a.n + FT - 1) / FT, (a.m + FT - 1) / FT), dim3(256), 0, st, a);
}

constexpr uint32_t MR_MAX_SMEM = 208 * 1024;
template <int PRO>
cudaError_t launch_fused(const MatvecSegs& p, uint32_t blocks, size_t smem, uint32_t* status, cudaStream_t st) {
    static PerDeviceFlag flag;
    if (const cudaError_t e = ensure_max_dynamic_smem(dense_matvec_kernel<PRO>, MR_MAX_SMEM, flag); e != cudaSuccess) return e;
    return launch_pdl(dense_matvec_kernel<PRO>, dim3(blocks), dim3(MR_THREADS), smem, st, p, status);
}

}  // namespace
}  // namespace hf2q

using namespace hf2q;

extern "C" {

HF2Q_API int32_t hf2q_cuda_dense_matmul(hf2q_ctx* ctx, void* stream, const void* x, uint32_t x_dtype, uint32_t ldx, const void* w, void* y,
                                        uint32_t y_dtype, uint32_t ldy, uint32_t m, uint32_t n, uint32_t k, uint32_t epilogue,
                                        const float* residual, float cap) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!x || !w || !y || n == 0 || k == 0 || k % 8 || ldx < k || ldy < n || reinterpret_cast<uintptr_t>(w) % 16)
        return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "dense_matmul: null pointer, k not a multiple of 8, a short row pitch or an unaligned weight");
    if (epilogue > HF2Q_EPI_SOFTCAP || (epilogue == HF2Q_EPI_ADD && !residual) || (epilogue == HF2Q_EPI_SOFTCAP && !(cap > 0.f)))
        return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "dense_matmul: bad epilogue");
    if (m == 0) return HF2Q_OK;
    if (m > 65535u * 64u) return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "dense_matmul: too many rows");
    const DenseArgs a{x, static_cast<const __nv_bfloat16*>(w), y, residual, ldx, ldy, m, n, k, epilogue, cap};
    const cudaStream_t st = static_cast<cudaStream_t>(stream);
    uint32_t* status = ctx_status_word(ctx);
    const int sms = ctx_sm_count(ctx);
    uint64_t launches = 0;
    cudaError_t e = cudaErrorInvalidValue;
    if (x_dtype == HF2Q_DT_F32 && y_dtype == HF2Q_DT_F32) e = dense_any<float, float>(a, sms, status, st, &launches);
    else if (x_dtype == HF2Q_DT_BF16 && y_dtype == HF2Q_DT_F32) e = dense_any<__nv_bfloat16, float>(a, sms, status, st, &launches);
    else if (x_dtype == HF2Q_DT_BF16 && y_dtype == HF2Q_DT_BF16) e = dense_any<__nv_bfloat16, __nv_bfloat16>(a, sms, status, st, &launches);
    else if (x_dtype == HF2Q_DT_F32 && y_dtype == HF2Q_DT_BF16) e = dense_any<float, __nv_bfloat16>(a, sms, status, st, &launches);
    return ctx_cuda_result(ctx, e, "dense_matmul", launches);
}

HF2Q_API int32_t hf2q_cuda_dense_matvec(hf2q_ctx* ctx, void* stream, uint32_t prologue, const hf2q_matvec* segs, uint32_t n_segs) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!segs || n_segs == 0 || n_segs > 2 || prologue > HF2Q_PRO_GATED) return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "dense_matvec: bad segments");
    MatvecSegs p{};
    uint32_t kmax = 0;
    uint64_t chunks[2] = {0, 0};
    for (uint32_t i = 0; i < n_segs; ++i) {
        const hf2q_matvec& s = segs[i];
        if (!s.w || !s.y || s.n == 0 || s.k == 0 || s.k % 8 || reinterpret_cast<uintptr_t>(s.w) % 16 || MR_RING + s.k * 4ull > MR_MAX_SMEM ||
            (prologue == HF2Q_PRO_NONE && !s.x) ||
            (prologue == HF2Q_PRO_NORM && (!s.pre.x || !s.pre.norm || s.pre.width > s.k || !pre_norm_aligned(s.pre) || (s.pre.a && (!s.pre.b || !s.pre.a_norm || !s.pre.b_norm)) || (s.pre.shift && (!s.pre.shift_state || !s.pre.pos)))) ||
            (prologue == HF2Q_PRO_GATED && (!s.gated.o || !s.gated.gate || s.gated.heads * s.gated.head_dim > s.k)) ||
            (s.epilogue == HF2Q_EPI_ADD && !s.residual))
            return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "dense_matvec: bad segment");
        p.s[i] = s;
        chunks[i] = static_cast<uint64_t>(s.n) * ((s.k + MV_CHUNK - 1) / MV_CHUNK);
        kmax = s.k > kmax ? s.k : kmax;
    }
    // one CTA per SM, shared by the segments in proportion to their chunks; no more CTAs than rows
    const uint64_t total = chunks[0] + chunks[1], sms = static_cast<uint64_t>(ctx_sm_count(ctx));
    auto ctas = [&](uint32_t i, uint64_t want) { return static_cast<uint32_t>(want < 1 ? 1 : want > segs[i].n ? segs[i].n : want); };
    uint32_t blocks = p.blocks0 = ctas(0, n_segs == 1 ? sms : (sms * chunks[0] + total / 2) / total);
    if (n_segs == 2) blocks += ctas(1, sms > p.blocks0 ? sms - p.blocks0 : 1);
    const cudaStream_t st = static_cast<cudaStream_t>(stream);
    const size_t smem = MR_RING + static_cast<size_t>(kmax) * 4;
    uint32_t* status = ctx_status_word(ctx);
    cudaError_t e;
    switch (prologue) {
        case HF2Q_PRO_NONE: e = launch_fused<HF2Q_PRO_NONE>(p, blocks, smem, status, st); break;
        case HF2Q_PRO_NORM: e = launch_fused<HF2Q_PRO_NORM>(p, blocks, smem, status, st); break;
        default: e = launch_fused<HF2Q_PRO_GATED>(p, blocks, smem, status, st); break;
    }
    return ctx_cuda_result(ctx, e, "dense_matvec", 1);
}

}  // extern "C"
