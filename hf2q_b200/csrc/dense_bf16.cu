// Products with bf16 weights: y[m][n] = epilogue(x[m][k] . w[n][k]^T), f32 accumulation.
//
//   dense_matvec_kernel   m = 1..8 rows; weights streamed with 16-byte loads, activations f32 in shared memory, fp32
//                         arithmetic (HBM-bound: 2 bytes per weight against one FMA per row).  With one row the
//                         layer's norm / token shift / gating runs in the kernel's own prologue.
//   dense_gemm_tc_kernel  more rows, bf16 activations: persistent tcgen05 kernel, both operands by TMA with 128-byte
//                         swizzle, two accumulator buffers in tensor memory so that the epilogue of a tile runs under
//                         the main loop of the next.
//   dense_gemm_f32_kernel more rows, f32 activations: CUDA-core tiles in full 32-bit arithmetic.
// Both take rows sorted by group (expert) with one weight matrix per group as well.
#include "matvec_stream.cuh"
#include "seq_common.cuh"
#include "tc_common.cuh"

namespace hf2q {
namespace {
using namespace seq;

__device__ __forceinline__ float epilogue_value(float v, uint32_t epi, float cap) {
    if (epi == HF2Q_EPI_GELU) return gelu_tanhf(v);
    if (epi == HF2Q_EPI_SOFTCAP) return cap * tanhf(v / cap);
    if (epi == HF2Q_EPI_SCALE) return v * cap;
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

// One-row product: the CTA's weight rows run through a MatvecStream; the layer's row prologue fills x in front of it.
template <int PRO, bool PAIRS>
__global__ void __launch_bounds__(MR_THREADS) dense_matvec_kernel(const __grid_constant__ MatvecSegs p, uint32_t* status) {
    extern __shared__ __align__(128) uint8_t mv_smem[];                 // ring, then x [k] f32
    __shared__ float red[64];
    __shared__ MatvecShared sh;
    pdl_trigger();
    const bool second = blockIdx.x >= p.blocks0;
    const hf2q_matvec& s = p.s[second];
    const uint32_t blk = blockIdx.x - (second ? p.blocks0 : 0u), n_blk = second ? gridDim.x - p.blocks0 : p.blocks0;
    const uint32_t warp = threadIdx.x >> 5;
    float* xs = reinterpret_cast<float*>(mv_smem + MR_RING);
    // rows [row0, row1) of this CTA, spread evenly
    constexpr uint32_t unit = PAIRS ? 2 : 1;
    const uint32_t units = s.n / unit;
    const uint32_t row0 = unit * static_cast<uint32_t>(static_cast<uint64_t>(units) * blk / n_blk), row1 = unit * static_cast<uint32_t>(static_cast<uint64_t>(units) * (blk + 1) / n_blk);
    const uint32_t per_row = (s.k + MV_CHUNK - 1) / MV_CHUNK;
    const __nv_bfloat16* w = static_cast<const __nv_bfloat16*>(s.w) + static_cast<size_t>(row0) * s.k;
    auto chunk = [&](uint32_t c) {
        const uint32_t k0 = (c % per_row) * MV_CHUNK;
        return MatvecChunk{w + static_cast<size_t>(c / per_row) * s.k + k0, k0, min(static_cast<uint32_t>(MV_CHUNK), s.k - k0)};
    };
    MatvecStream stream(mv_smem, sh, (row1 - row0) * per_row, status);
    stream.start(chunk);
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
    } else if constexpr (PRO == HF2Q_PRO_HYPER) {
        const hf2q_hyper& q = s.hyper;
        __shared__ float coef[HYPER_COEF];
        // every CTA makes the whole row and stores its share of the new streams
        const uint32_t lo = static_cast<uint32_t>(static_cast<uint64_t>(q.width) * blk / n_blk) & ~3u;
        const uint32_t hi = blk + 1 == n_blk ? q.width : static_cast<uint32_t>(static_cast<uint64_t>(q.width) * (blk + 1) / n_blk) & ~3u;
        const float inv = hyper_row(q, 0, xs, coef, red, lo, hi);
        for (uint32_t i = threadIdx.x; i < s.k; i += MR_THREADS) {
            const float h = i < q.width ? (q.norm ? xs[i] * inv * q.norm[i] : xs[i]) : 0.f;
            xs[i] = h;
            if (q.h_out && i >= lo && i < hi) q.h_out[i] = h;
        }
    } else {
        for (uint32_t i = s.gated.heads * s.gated.head_dim + threadIdx.x; i < s.k; i += MR_THREADS) xs[i] = 0.f;
        if (s.gated.kind == HF2Q_GATE_SILU_FIRST) silu_group_norm_row<float>(s.gated, 0, xs, xs);
        else gated_heads_row<float>(s.gated, 0, xs, warp, MR_WARPS);
    }
    __syncthreads();
    if constexpr (PAIRS) {
        stream.run<true>(chunk, xs, row1 - row0, per_row, [&](uint32_t r, float gate, float up) {
            const uint32_t row = row0 + r;
            if (s.bias) { gate += s.bias[row]; up += s.bias[row + 1]; }
            s.y[row / 2] = glu_value(gate, up, s.epilogue, s.cap);
        });
    } else {
        stream.run<false>(chunk, xs, row1 - row0, per_row, [&](uint32_t r, float v, float) {
            const uint32_t row = row0 + r;
            if (s.bias) v += s.bias[row];
            v = epilogue_value(v, s.epilogue, s.cap);
            if (s.epilogue == HF2Q_EPI_ADD) v += s.residual[row];
            s.y[row] = v;
        });
    }
}

struct DenseArgs {
    const void* x;
    const __nv_bfloat16* w;
    void* y;
    const float *residual, *bias;
    uint32_t ldx, ldy, m, n, k, epi;
    float cap;
    hf2q_row_groups g;       // grouped products: rows of x sorted by group, w [groups][n][k]
};
// where a grouped product's output row goes, and what it is scaled with before the activation
struct GroupRow { size_t out; float scale; };
__device__ __forceinline__ GroupRow group_row(const DenseArgs& p, uint32_t sorted) {
    const uint32_t routed = p.g.perm[sorted];
    return {p.g.scatter ? routed : sorted, p.g.row_scale ? p.g.row_scale[routed] : 1.0f};
}

template <typename X, typename Y, int M, int RW>
__global__ void __launch_bounds__(MV_THREADS) dense_matvec_m_kernel(const DenseArgs p) {          // RW = 2: rows are pairs
    extern __shared__ __align__(16) float xs[];
    pdl_trigger();
    pdl_wait();
    const X* x = static_cast<const X*>(p.x);
    for (int m = 0; m < M; ++m)
        for (uint32_t i = threadIdx.x; i < p.k; i += MV_THREADS)
            xs[static_cast<size_t>(m) * p.k + i] = m < static_cast<int>(p.m) ? to_f32(x[static_cast<size_t>(m) * p.ldx + i]) : 0.f;
    __syncthreads();
    const uint32_t row = (blockIdx.x * MV_WARPS + (threadIdx.x >> 5)) * RW;
    if (row >= p.n) return;
    float acc[RW][M];
#pragma unroll
    for (int r = 0; r < RW; ++r)
#pragma unroll
        for (int m = 0; m < M; ++m) acc[r][m] = 0.f;
    matvec_rows<RW, M>(p.w, row, p.n, p.k, xs, acc);
    if ((threadIdx.x & 31) == 0) {
#pragma unroll
        for (int m = 0; m < M; ++m)
            if (m < static_cast<int>(p.m)) {
                const size_t o = static_cast<size_t>(m) * p.ldy + row / RW;
                float v = acc[0][m] + (p.bias ? p.bias[row] : 0.f);
                if constexpr (RW == 2) {
                    v = glu_value(v, acc[1][m] + (p.bias ? p.bias[row + 1] : 0.f), p.epi, p.cap);
                } else {
                    v = epilogue_value(v, p.epi, p.cap);
                    if (p.epi == HF2Q_EPI_ADD) v += p.residual[o];
                }
                static_cast<Y*>(p.y)[o] = from_f32<Y>(v);
            }
    }
}

// ---------------------------------------------------------------- fp32 product on the CUDA cores
constexpr int FT = 64, FK = 16;

template <typename X, typename Y, bool GROUPED>
__global__ void __launch_bounds__(256) dense_gemm_f32_kernel(const DenseArgs p) {
    __shared__ float as[FK][FT + 4], bs[FK][FT + 4];
    pdl_trigger();
    pdl_wait();
    const X* x = static_cast<const X*>(p.x);
    uint32_t m0 = blockIdx.y * FT, m_end = p.m;
    const uint32_t n0 = blockIdx.x * FT;
    const __nv_bfloat16* w = p.w;
    if constexpr (GROUPED) {
        if (blockIdx.y >= p.g.header[0]) return;
        const uint4 tile = reinterpret_cast<const uint4*>(p.g.tiles)[blockIdx.y];           // group, first sorted row, rows
        w += static_cast<size_t>(tile.x) * p.n * p.k;
        m0 = tile.y;
        m_end = tile.y + tile.z;
    }
    const uint32_t tr = threadIdx.x / 16, tc = threadIdx.x % 16;
    float acc[4][4] = {};
    for (uint32_t k0 = 0; k0 < p.k; k0 += FK) {
        for (uint32_t i = threadIdx.x; i < FT * FK; i += 256) {
            const uint32_t r = i / FK, c = i % FK;
            as[c][r] = m0 + r < m_end && k0 + c < p.k ? to_f32(x[static_cast<size_t>(m0 + r) * p.ldx + k0 + c]) : 0.f;
            bs[c][r] = n0 + r < p.n && k0 + c < p.k ? to_f32(w[static_cast<size_t>(n0 + r) * p.k + k0 + c]) : 0.f;
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
    const bool pairs = epi_pairs(p.epi);
    for (int i = 0; i < 4; ++i) {
        const uint32_t r = m0 + 4 * tr + i;
        if (r >= m_end) continue;
        size_t row = r;
        float scale = 1.0f;
        if constexpr (GROUPED) { const GroupRow q = group_row(p, r); row = q.out; scale = q.scale; }
        for (int j = 0; j < 4; ++j) {
            const uint32_t c = n0 + 4 * tc + j;
            if (c >= p.n || (pairs && (j & 1))) continue;
            const size_t o = row * p.ldy + (pairs ? c / 2 : c);
            float v = acc[i][j] * scale + (p.bias ? p.bias[c] : 0.f);
            if (pairs) {
                v = glu_value(v, acc[i][j + 1 < 4 ? j + 1 : j] * scale + (p.bias ? p.bias[c + 1] : 0.f), p.epi, p.cap);
            } else {
                v = epilogue_value(v, p.epi, p.cap);
                if (p.epi == HF2Q_EPI_ADD) v += p.residual[o];
            }
            static_cast<Y*>(p.y)[o] = from_f32<Y>(v);
        }
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

// sixteen consecutive outputs, 32-byte aligned for f32 and 16-byte aligned for bf16
__device__ __forceinline__ void store16(float* y, const float* v) {
    st_global_v8(y, v);
    st_global_v8(y + 8, v + 8);
}
__device__ __forceinline__ void store16(__nv_bfloat16* y, const float* v) {
    uint32_t q[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
        const __nv_bfloat162 h = __floats2bfloat162_rn(v[2 * j], v[2 * j + 1]);
        q[j] = *reinterpret_cast<const uint32_t*>(&h);
    }
    reinterpret_cast<uint4*>(y)[0] = make_uint4(q[0], q[1], q[2], q[3]);
    reinterpret_cast<uint4*>(y)[1] = make_uint4(q[4], q[5], q[6], q[7]);
}

template <int NT, typename Y, bool GROUPED>
__global__ void __launch_bounds__(TC_THREADS, 1) dense_gemm_tc_kernel(const __grid_constant__ CUtensorMap map_x, const __grid_constant__ CUtensorMap map_w,
                                                                      const DenseArgs p, uint32_t* status) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
    constexpr int ST = tc_stages(NT);
    constexpr uint32_t SB = tc_stage_bytes(NT);
    __shared__ uint64_t full[ST], empty[ST], d_full[2], d_empty[2];
    __shared__ uint32_t tmem_slot;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t nkb = (p.k + TC_K - 1) / TC_K;
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
    const uint32_t mt = GROUPED ? p.g.header[0] : (p.m + TC_M - 1) / TC_M, n_tiles = mt * ((p.n + NT - 1) / NT);
    const uint4* group_tiles = reinterpret_cast<const uint4*>(p.g.tiles);                // group, first sorted row, rows
    if (warp == 0) {
        if (lane == 0) {
            uint32_t it = 0;
            bool ok = true;
            for (uint32_t tile = blockIdx.x; tile < n_tiles && ok; tile += gridDim.x) {
                int row_x = static_cast<int>((tile % mt) * TC_M), row_w = static_cast<int>((tile / mt) * NT);
                if constexpr (GROUPED) {
                    const uint4 q = group_tiles[tile % mt];
                    row_x = static_cast<int>(q.y);
                    row_w += static_cast<int>(q.x * p.n);
                }
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
            const uint32_t n0 = (tile / mt) * NT, n_cols = min(static_cast<uint32_t>(NT), p.n - n0);
            size_t row = (tile % mt) * TC_M + quad * 32 + lane;
            bool live = row < p.m;
            float scale = 1.0f;
            if constexpr (GROUPED) {
                const uint4 q = group_tiles[tile % mt];
                live = quad * 32 + lane < q.z;
                if (live) { const GroupRow gr = group_row(p, q.y + quad * 32 + lane); row = gr.out; scale = gr.scale; }
            }
#pragma unroll 1
            for (uint32_t c0 = 0; c0 < n_cols; c0 += 32) {
                uint32_t r[32];
                tc::tmem_ld32(tmem + b * NT + ((quad * 32u) << 16) + c0, r);
                tc::tmem_wait_ld();
                if (live) {
                float v[32];
#pragma unroll
                for (int j = 0; j < 32; ++j) v[j] = __uint_as_float(r[j]);
                if constexpr (GROUPED) {
#pragma unroll
                    for (int j = 0; j < 32; ++j) v[j] *= scale;
                }
                if (p.bias) {
#pragma unroll
                    for (int j = 0; j < 32; ++j)
                        if (c0 + j < n_cols) v[j] += p.bias[n0 + c0 + j];
                }
                if (epi_pairs(p.epi)) {                                  // 32 columns -> 16 outputs
                    Y* y = static_cast<Y*>(p.y) + row * p.ldy + (n0 + c0) / 2;
                    float g[16];
#pragma unroll
                    for (int j = 0; j < 16; ++j) g[j] = glu_value(v[2 * j], v[2 * j + 1], p.epi, p.cap);
                    if (wide && c0 + 32 <= n_cols) {
                        store16(y, g);
                    } else {
#pragma unroll
                        for (int j = 0; j < 16; ++j)
                            if (c0 + 2 * j < n_cols) y[j] = from_f32<Y>(g[j]);
                    }
                } else {
                const size_t o = row * p.ldy + n0 + c0;
                Y* y = static_cast<Y*>(p.y) + o;
                if (p.epi == HF2Q_EPI_GELU || p.epi == HF2Q_EPI_SOFTCAP || p.epi == HF2Q_EPI_SCALE) {
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
                    store16(y, v);
                    store16(y + 16, v + 16);
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

template <int NT, typename Y, bool GROUPED>
cudaError_t launch_tc(const DenseArgs& a, uint32_t m_tiles, int sms, uint32_t* status, cudaStream_t st) {
    CUtensorMap mx, mw;
    const uint32_t w_rows = GROUPED ? a.n * a.g.groups : a.n;
    if (!encode_rows(&mx, a.x, a.m, a.k, a.ldx, TC_M) || !encode_rows(&mw, a.w, w_rows, a.k, a.k, NT)) return cudaErrorInvalidValue;
    const size_t smem = 1024 + static_cast<size_t>(tc_stages(NT)) * tc_stage_bytes(NT);
    static PerDeviceFlag flag;
    if (const cudaError_t e = ensure_max_dynamic_smem(dense_gemm_tc_kernel<NT, Y, GROUPED>, static_cast<int>(smem), flag); e != cudaSuccess) return e;
    const uint32_t tiles = m_tiles * ((a.n + NT - 1) / NT);
    const uint32_t grid = tiles < static_cast<uint32_t>(sms) ? tiles : static_cast<uint32_t>(sms);
    return launch_pdl(dense_gemm_tc_kernel<NT, Y, GROUPED>, dim3(grid), dim3(TC_THREADS), smem, st, mx, mw, a, status);
}
// m_tiles: activation tiles, for a grouped product the most there can be
template <typename Y, bool GROUPED>
cudaError_t launch_tc_any(const DenseArgs& a, uint32_t m_tiles, int sms, uint32_t* status, cudaStream_t st) {
    // the widest tile that still gives (nearly) every SM work
    if (m_tiles * ((a.n + 255) / 256) >= static_cast<uint32_t>(sms) * 3 / 4) return launch_tc<256, Y, GROUPED>(a, m_tiles, sms, status, st);
    if (m_tiles * ((a.n + 127) / 128) >= static_cast<uint32_t>(sms) * 3 / 4) return launch_tc<128, Y, GROUPED>(a, m_tiles, sms, status, st);
    return launch_tc<64, Y, GROUPED>(a, m_tiles, sms, status, st);
}

constexpr uint32_t MV_SMEM = 200 * 1024;

template <typename X, typename Y, int M, int RW>
cudaError_t launch_mv_rw(const DenseArgs& a, cudaStream_t st) {
    static PerDeviceFlag flag;
    if (const cudaError_t e = ensure_max_dynamic_smem(dense_matvec_m_kernel<X, Y, M, RW>, MV_SMEM, flag); e != cudaSuccess) return e;
    return launch_pdl(dense_matvec_m_kernel<X, Y, M, RW>, dim3((a.n / RW + MV_WARPS - 1) / MV_WARPS), dim3(MV_THREADS),
                      static_cast<size_t>(M) * a.k * 4, st, a);
}
template <typename X, typename Y, int M>
cudaError_t launch_mv_m(const DenseArgs& a, cudaStream_t st) {
    return epi_pairs(a.epi) ? launch_mv_rw<X, Y, M, 2>(a, st) : launch_mv_rw<X, Y, M, 1>(a, st);
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
        if (a.ldx % 8 == 0 && reinterpret_cast<uintptr_t>(a.x) % 16 == 0) return launch_tc_any<Y, false>(a, (a.m + TC_M - 1) / TC_M, sms, status, st);
    }
    return launch_pdl(dense_gemm_f32_kernel<X, Y, false>, dim3((a.n + FT - 1) / FT, (a.m + FT - 1) / FT), dim3(256), 0, st, a);
}

template <int PRO, bool PAIRS>
cudaError_t launch_fused_as(const MatvecSegs& p, uint32_t blocks, size_t smem, uint32_t* status, cudaStream_t st) {
    static PerDeviceFlag flag;
    if (const cudaError_t e = ensure_max_dynamic_smem(dense_matvec_kernel<PRO, PAIRS>, MR_MAX_SMEM, flag); e != cudaSuccess) return e;
    return launch_pdl(dense_matvec_kernel<PRO, PAIRS>, dim3(blocks), dim3(MR_THREADS), smem, st, p, status);
}
template <int PRO>
cudaError_t launch_fused(const MatvecSegs& p, uint32_t blocks, size_t smem, uint32_t* status, cudaStream_t st) {
    return epi_pairs(p.s[0].epilogue) ? launch_fused_as<PRO, true>(p, blocks, smem, status, st) : launch_fused_as<PRO, false>(p, blocks, smem, status, st);
}

}  // namespace
}  // namespace hf2q

using namespace hf2q;

extern "C" {

HF2Q_API int32_t hf2q_cuda_dense_matmul(hf2q_ctx* ctx, void* stream, const void* x, uint32_t x_dtype, uint32_t ldx, const void* w, void* y,
                                        uint32_t y_dtype, uint32_t ldy, uint32_t m, uint32_t n, uint32_t k, uint32_t epilogue,
                                        const float* residual, float cap, const float* bias) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!x || !w || !y || n == 0 || k == 0 || k % 8 || ldx < k || ldy < (epi_pairs(epilogue) ? n / 2 : n) || reinterpret_cast<uintptr_t>(w) % 16)
        return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "dense_matmul: null pointer, k not a multiple of 8, a short row pitch or an unaligned weight");
    if (epilogue > HF2Q_EPI_CLAMP_GLU || (epilogue == HF2Q_EPI_ADD && !residual) || (epi_needs_cap(epilogue) && !(cap > 0.f)) || (epi_pairs(epilogue) && n % 2))
        return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "dense_matmul: bad epilogue");
    if (m == 0) return HF2Q_OK;
    if (m > 65535u * 64u) return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "dense_matmul: too many rows");
    const DenseArgs a{x, static_cast<const __nv_bfloat16*>(w), y, residual, bias, ldx, ldy, m, n, k, epilogue, cap, {}};
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

HF2Q_API int32_t hf2q_cuda_dense_grouped(hf2q_ctx* ctx, void* stream, const hf2q_row_groups* g, const void* x, uint32_t dtype, uint32_t ldx, const void* w,
                                         void* y, uint32_t y_dtype, uint32_t ldy, uint32_t rows, uint32_t n, uint32_t k, uint32_t epilogue, float cap) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!g || !g->header || !g->tiles || !g->perm || g->groups == 0 || !x || !w || !y || n == 0 || k == 0 || k % 8 || ldx < k || ldx % 8 ||
        ldy < (epi_pairs(epilogue) ? n / 2 : n) || reinterpret_cast<uintptr_t>(w) % 16 || reinterpret_cast<uintptr_t>(x) % 16 || epilogue > HF2Q_EPI_CLAMP_GLU ||
        epilogue == HF2Q_EPI_ADD || (epi_needs_cap(epilogue) && !(cap > 0.f)) || (epi_pairs(epilogue) && n % 2) || static_cast<uint64_t>(g->groups) * n > 0x7fffffffu)
        return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "dense_grouped: null or unaligned pointer, or a bad size or epilogue");
    if (rows == 0) return HF2Q_OK;
    if (g->tile_rows != (dtype == HF2Q_DT_BF16 ? HF2Q_GROUP_TILE_BF16 : HF2Q_GROUP_TILE_F32))
        return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "dense_grouped: the rows were sorted for another tile height");
    DenseArgs a{x, static_cast<const __nv_bfloat16*>(w), y, nullptr, nullptr, ldx, ldy, rows, n, k, epilogue, cap, *g};
    const cudaStream_t st = static_cast<cudaStream_t>(stream);
    const uint32_t most = rows / g->tile_rows + (rows < g->groups ? rows : g->groups);     // sum of ceil(count / tile_rows)
    cudaError_t e = cudaErrorInvalidValue;
    if (dtype == HF2Q_DT_BF16 && y_dtype == HF2Q_DT_BF16) e = launch_tc_any<__nv_bfloat16, true>(a, most, ctx_sm_count(ctx), ctx_status_word(ctx), st);
    else if (dtype == HF2Q_DT_BF16 && y_dtype == HF2Q_DT_F32) e = launch_tc_any<float, true>(a, most, ctx_sm_count(ctx), ctx_status_word(ctx), st);
    else if (dtype == HF2Q_DT_F32 && y_dtype == HF2Q_DT_F32 && most <= 65535)
        e = launch_pdl(dense_gemm_f32_kernel<float, float, true>, dim3((n + FT - 1) / FT, most), dim3(256), 0, st, a);
    return ctx_cuda_result(ctx, e, "dense_grouped", 1);
}

HF2Q_API int32_t hf2q_cuda_dense_matvec(hf2q_ctx* ctx, void* stream, uint32_t prologue, const hf2q_matvec* segs, uint32_t n_segs) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!segs || n_segs == 0 || n_segs > 2 || prologue > HF2Q_PRO_HYPER) return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "dense_matvec: bad segments");
    MatvecSegs p{};
    uint32_t kmax = 0;
    uint64_t chunks[2] = {0, 0};
    for (uint32_t i = 0; i < n_segs; ++i) {
        const hf2q_matvec& s = segs[i];
        if (!s.w || !s.y || s.n == 0 || s.k == 0 || s.k % 8 || reinterpret_cast<uintptr_t>(s.w) % 16 || MR_RING + s.k * 4ull > MR_MAX_SMEM ||
            (prologue == HF2Q_PRO_NONE && !s.x) ||
            (prologue == HF2Q_PRO_NORM && (!s.pre.x || !s.pre.norm || s.pre.width > s.k || !pre_norm_aligned(s.pre) || (s.pre.a && (!s.pre.b || !s.pre.a_norm || !s.pre.b_norm)) || (s.pre.shift && (!s.pre.shift_state || !s.pre.pos)))) ||
            (prologue == HF2Q_PRO_GATED && (!gated_ok(s.gated) || s.gated.heads * s.gated.head_dim > s.k)) ||
            (prologue == HF2Q_PRO_HYPER && (!hyper_ok(s.hyper) || s.hyper.width > s.k || s.hyper.x_out == s.hyper.x)) || s.epilogue > HF2Q_EPI_CLAMP_GLU ||
            (s.epilogue == HF2Q_EPI_ADD && !s.residual) || (epi_needs_cap(s.epilogue) && !(s.cap > 0.f)) || (epi_pairs(s.epilogue) && s.n % 2) || epi_pairs(s.epilogue) != epi_pairs(segs[0].epilogue))
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
        case HF2Q_PRO_HYPER: e = launch_fused<HF2Q_PRO_HYPER>(p, blocks, smem, status, st); break;
        default: e = launch_fused<HF2Q_PRO_GATED>(p, blocks, smem, status, st); break;
    }
    return ctx_cuda_result(ctx, e, "dense_matvec", 1);
}

}  // extern "C"
