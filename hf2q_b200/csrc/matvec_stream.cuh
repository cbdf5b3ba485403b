// Weight stream of the one-row products: a CTA's weights are cut into chunks of MV_CHUNK elements; its warps take the
// chunks in turn, each through a private ring of bulk copies.  Where the addresses do not depend on an earlier kernel the
// ring starts filling before the wait for it (weights never change).  Chunk sums of a block of rows meet in shared memory
// and are added in chunk order.
#pragma once
#include "seq_common.cuh"

namespace hf2q {
namespace seq {

constexpr int MR_WARPS = 16, MR_THREADS = MR_WARPS * 32, MV_CHUNK = 1024, MR_STAGES = 3, MR_PART = 2048;
constexpr uint32_t MR_RING = MR_WARPS * MR_STAGES * MV_CHUNK * 2;      // bytes of dynamic shared memory
constexpr uint32_t MR_MAX_SMEM = 208 * 1024;

struct MatvecShared {
    float part[2][MR_PART];
    uint64_t bars[MR_WARPS][MR_STAGES];
};
struct MatvecChunk {
    const __nv_bfloat16* w;      // global, 16-byte aligned
    uint32_t x0, len;            // its activations start at xs + x0; len a multiple of 8
};

class MatvecStream {
public:
    __device__ __forceinline__ MatvecStream(uint8_t* smem, MatvecShared& sh, uint32_t n_chunks, uint32_t* status)
        : sh_(sh), n_chunks_(n_chunks), status_(status), warp_(threadIdx.x >> 5), lane_(threadIdx.x & 31),
          ring_(reinterpret_cast<__nv_bfloat16*>(smem) + static_cast<size_t>(warp_) * MR_STAGES * MV_CHUNK) {}

    // fills the ring; chunk(c) -> MatvecChunk
    template <class F> __device__ __forceinline__ void start(F chunk) {
        if (lane_ == 0) {
            for (int i = 0; i < MR_STAGES; ++i) mbar_init(&sh_.bars[warp_][i], 1);
            mbar_fence_init();
            for (int i = 0; i < MR_STAGES; ++i) issue(i, chunk);
        }
    }
    // rows of per_row chunks each, finished one (or with PAIRS two) at a time: finish(row, sum, sum of row + 1).  Every thread
    // of the CTA calls it, after a barrier behind the last write of xs.
    template <bool PAIRS, class F, class G> __device__ __forceinline__ void run(F chunk, const float* xs, uint32_t rows, uint32_t per_row, G finish) {
        constexpr uint32_t unit = PAIRS ? 2 : 1;
        const uint32_t block_rows = max(unit, MR_PART / per_row / unit * unit);
        bool ok = true;
        uint32_t i = 0;                                                     // this warp's chunk counter
        for (uint32_t r0 = 0, pb = 0; r0 < rows; r0 += block_rows, pb ^= 1) {
            const uint32_t nr = min(block_rows, rows - r0), c_end = (r0 + nr) * per_row;
            for (uint32_t c = i * MR_WARPS + warp_; c < c_end; ++i, c += MR_WARPS) {
                const uint32_t st = i % MR_STAGES;
                const MatvecChunk k = chunk(c);
                if (ok) ok = mbar_wait_bounded(&sh_.bars[warp_][st], (i / MR_STAGES) & 1, status_);
                ok = __all_sync(0xffffffffu, ok);
                float acc = 0.f;
                if (ok) {
                    const uint4* wv = reinterpret_cast<const uint4*>(ring_ + st * MV_CHUNK);
                    const float* xv = xs + k.x0;
#pragma unroll
                    for (int u = 0; u < MV_CHUNK / 256; ++u) {
                        const uint32_t e = lane_ + 32 * u;
                        if (8 * e < k.len) {
                            const uint4 v = wv[e];
                            const float4 a = *reinterpret_cast<const float4*>(xv + 8 * e), b = *reinterpret_cast<const float4*>(xv + 8 * e + 4);
                            acc = fmaf(bf_lo(v.x), a.x, acc); acc = fmaf(bf_hi(v.x), a.y, acc); acc = fmaf(bf_lo(v.y), a.z, acc); acc = fmaf(bf_hi(v.y), a.w, acc);
                            acc = fmaf(bf_lo(v.z), b.x, acc); acc = fmaf(bf_hi(v.z), b.y, acc); acc = fmaf(bf_lo(v.w), b.z, acc); acc = fmaf(bf_hi(v.w), b.w, acc);
                        }
                    }
                }
                __syncwarp();                                               // every lane has read the stage
                if (lane_ == 0 && ok) issue(i + MR_STAGES, chunk);
                acc = warp_sum(acc);
                if (lane_ == 0) sh_.part[pb][c - r0 * per_row] = acc;
            }
            __syncthreads();                                                // (the other half of `part` is free: its readers passed this barrier)
            for (uint32_t r = threadIdx.x * unit; r < nr; r += MR_THREADS * unit) {
                float v = 0.f, w = 0.f;
                for (uint32_t kc = 0; kc < per_row; ++kc) v += sh_.part[pb][r * per_row + kc];
                if constexpr (PAIRS)
                    for (uint32_t kc = 0; kc < per_row; ++kc) w += sh_.part[pb][(r + 1) * per_row + kc];
                finish(r0 + r, v, w);
            }
        }
    }

private:
    template <class F> __device__ __forceinline__ void issue(uint32_t i, F& chunk) {      // this warp's chunk number i
        const uint32_t c = i * MR_WARPS + warp_;
        if (c >= n_chunks_) return;
        const MatvecChunk k = chunk(c);
        uint64_t* bar = &sh_.bars[warp_][i % MR_STAGES];
        mbar_arrive_expect_tx(bar, k.len * 2);
        bulk_g2s(ring_ + (i % MR_STAGES) * MV_CHUNK, k.w, k.len * 2, bar);
    }
    MatvecShared& sh_;
    const uint32_t n_chunks_;
    uint32_t* const status_;
    const uint32_t warp_, lane_;
    __nv_bfloat16* const ring_;
};

}  // namespace seq
}  // namespace hf2q
